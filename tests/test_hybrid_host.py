"""Host side of the hybrid decoder and of the engine, without a GPU: configuration, checkpoint reading, registry, page and
slot bookkeeping, step metadata, scheduling (over a model that is a plain function) and trace replay."""

import io
import json

import pytest
import torch

import plain_hybrid as plain
import vllm_rlt_b200 as rlt
from hybrid_cases import CONFIGS, attention_layer, make_config, mamba_layer, prompt, random_weights, write_model, write_safetensors
from vllm_rlt_b200 import engine as engine_module
from vllm_rlt_b200 import hybrid_lm, registry, trace
from vllm_rlt_b200.runner import Request, SamplingParams


# ---- configuration and weights -------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configurations_parse_and_name_every_tensor(name):
    config = rlt.HybridLMConfig.from_json(CONFIGS[name])
    weights = random_weights(hybrid_lm.parameter_shapes(config), 0)
    model = rlt.HybridLM(config, weights, "cpu")
    for i, (layer, entry) in enumerate(zip(model.layers, CONFIGS[name]["layers"])):
        assert layer.ff == (entry["mlp"]["ff"] if entry["mlp"] else 0)
        assert layer.w_in.shape[0] % 8 == 0 and layer.operand_width % 8 == 0
        if entry["type"] == "attention" and "kv_from" in entry["mixer"]:
            assert f"l{i}.mix.k" not in weights and i not in model.cache_spec().layers


def test_stacked_projections_hold_the_weights_at_their_columns():
    config = rlt.HybridLMConfig.from_json(CONFIGS["odd"])
    weights = random_weights(hybrid_lm.parameter_shapes(config), 1)
    layer = rlt.HybridLM(config, weights, "cpu").layers[1]
    for name, at in (("q", 0), ("k", layer.k_col), ("v", layer.v_col)):
        w = weights["l1.mix." + name]
        assert torch.equal(layer.w_in[at:at + w.shape[0]], w)
    assert torch.equal(layer.w_in[layer.up_col:layer.up_col + layer.ff], weights["l1.mlp.up"])
    assert torch.equal(layer.w_out[:, :layer.inner], weights["l1.mix.o"])
    assert torch.equal(layer.w_out[:, layer.act_col:layer.act_col + layer.ff], weights["l1.mlp.down"])
    assert int(layer.w_out.count_nonzero()) <= weights["l1.mix.o"].numel() + weights["l1.mlp.down"].numel()


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0]["mixer"].update(window=5), "unknown config keys"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "lacks"),
    (lambda c: c["layers"][0].update(type="conv"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=8), "other key/value sizes"),
    (lambda c: c["layers"][1]["mixer"].update(groups=4), "multiple"),
    (lambda c: c["layers"][0]["mlp"].update(kind="router"), "feed-forward"),
    (lambda c: c.update(width=0), "width"),
])
def test_configurations_that_make_no_sense_are_refused(change, message):
    config = json.loads(json.dumps(CONFIGS["mixed"]))
    change(config)
    with pytest.raises(ValueError, match=message):
        rlt.HybridLMConfig.from_json(config)


def test_weights_of_another_shape_are_refused():
    config = rlt.HybridLMConfig.from_json(CONFIGS["odd"])
    weights = random_weights(hybrid_lm.parameter_shapes(config), 0)
    weights["l1.mix.v"] = weights["l1.mix.v"][:-1]
    with pytest.raises(ValueError, match="l1.mix.v"):
        rlt.HybridLM(config, weights, "cpu")
    del weights["l1.mix.v"]
    with pytest.raises(ValueError, match="lacks"):
        rlt.HybridLM(config, weights, "cpu")


def test_safetensors_files_are_read_back(tmp_path):
    tensors = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, 1, 4), "odd": torch.randn(3).bfloat16(),
               "after": torch.randn(2, 2)}
    write_safetensors(tmp_path / "model.safetensors", tensors)
    got = rlt.read_weights(tmp_path)
    assert set(got) == set(tensors) and all(torch.equal(got[k], v) and got[k].dtype == v.dtype for k, v in tensors.items())
    data = bytearray((tmp_path / "model.safetensors").read_bytes())
    (tmp_path / "short.safetensors").write_bytes(data[:-3])
    with pytest.raises(ValueError, match="byte range"):
        rlt.read_safetensors(tmp_path / "short.safetensors")


def test_the_registry_chooses_by_architecture(tmp_path):
    assert {"Sobipel", "OuroForCausalLM"} <= set(rlt.registered_architectures())
    assert registry.resolve({"architectures": ["OuroForCausalLM"]}).model_class is rlt.LoopedLM
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.resolve({"architecture": "Nothing"})
    config = rlt.HybridLMConfig.from_json(CONFIGS["odd"])
    write_model(tmp_path, CONFIGS["odd"], random_weights(hybrid_lm.parameter_shapes(config), 0))
    model = rlt.load_model(tmp_path, device="cpu", dtype=torch.float32)
    assert isinstance(model, rlt.HybridLM) and model.config == config and model.embed.dtype == torch.float32
    looped = rlt.LoopedLMConfig.from_json({"hidden_size": 64, "num_attention_heads": 4, "vocab_size": 9, "torch_dtype": "bfloat16"})
    assert (looped.head_dim, looped.vocab_size, looped.total_ut_steps) == (16, 9, 4)


# ---- pages and slots -----------------------------------------------------------------------------
def test_pages_and_slots_change_hands():
    spec = rlt.CacheSpec(planes=2, layers={0: rlt.KVSpec(1, 4, 6)}, states={"s": rlt.StateSpec((3,), torch.float32)})
    cache = rlt.SequenceCache(spec, max_tokens=96, max_sequences=2, device="cpu")
    assert cache.num_pages == 12 and cache.state["s"].shape == (3, 3) and cache.value[0].shape == (12, 16, 1, 6)
    cache.admit("a")
    cache.reserve("a", 33)
    assert [len(cache.pages("a", p)) for p in (0, 1)] == [3, 3] and not set(cache.pages("a", 0)) & set(cache.pages("a", 1))
    cache.reserve("a", 48)
    assert cache.free_pages == 6
    cache.admit("b")
    with pytest.raises(rlt.CacheFull):
        cache.admit("c")
    with pytest.raises(rlt.CacheFull):
        cache.reserve("b", 49)
    assert cache.pages("b") == [] and cache.free_pages == 6
    held, slot = cache.pages("a", 0) + cache.pages("a", 1), cache.slot("a")
    cache.release("a")
    cache.admit("c")
    cache.reserve("c", 48)
    assert cache.slot("c") == slot and set(cache.pages("c", 0) + cache.pages("c", 1)) == set(held)


# ---- the engine over a model that is a function --------------------------------------------------
class CountingModel:
    """Next token = (7 * sum of the sequence so far + length) mod vocab, computed from what the engine hands over: the
    running sums live in a state slot, the tokens themselves in 'pages', so wrong metadata shows in the output."""

    vocab_size, device, dtype = 53, torch.device("cpu"), torch.float32

    def cache_spec(self):
        return rlt.CacheSpec(layers={0: rlt.KVSpec(1, 1, 1)}, states={"sum": rlt.StateSpec((1,), torch.float32)})

    def forward_step(self, batch, cache):
        self.last = batch
        hidden = torch.zeros(batch.rows)
        covered = 0
        for group in batch.groups:
            assert torch.equal(group.cu - group.cu[0], group.local_cu) and group.rows.start == covered
            covered = group.rows.stop
            for s in range(group.sequences):
                lo, hi = int(group.cu[s]), int(group.cu[s + 1])
                start, slot = int(group.starts[s]), int(group.slots[s])
                assert hi - lo <= group.max_new and int(group.lengths[s]) == start + hi - lo
                total = 0.0 if start == 0 else float(cache.state["sum"][slot])
                for row in range(lo, hi):
                    position = start + row - lo
                    assert int(batch.positions[row]) == position
                    table = batch.tables[0, int(batch.row_seq[row])]
                    cache.key[0][table[position // cache.block], position % cache.block] = float(batch.tokens[row])
                    total += float(batch.tokens[row])
                    stored = sum(float(cache.key[0][table[p // cache.block], p % cache.block]) for p in range(position + 1))
                    assert stored == total
                    hidden[row] = (7 * total + position + 1) % self.vocab_size
                cache.state["sum"][slot] = total
        assert covered == batch.rows
        return hidden

    def step_logits(self, hidden, rows=None):
        picked = hidden if rows is None else hidden[rows]
        return torch.nn.functional.one_hot(picked.long(), self.vocab_size).float()


def expected_output(tokens, count):
    out = list(tokens)
    for _ in range(count):
        out.append((7 * sum(out) + len(out)) % CountingModel.vocab_size)
    return out[len(tokens):]


@pytest.fixture
def counting_engine(monkeypatch):
    monkeypatch.setattr(engine_module, "argmax_rows", lambda logits: logits.argmax(-1))

    def build(**kw):
        return rlt.Engine(CountingModel(), cuda_graphs=False, **{"max_tokens": 256, "max_sequences": 3, **kw})

    return build


def test_steps_mix_portions_and_single_tokens(counting_engine):
    engine = counting_engine()
    a, b = prompt(1, 60, 53), prompt(2, 45, 53)
    engine.step([dict(name="a", tokens=a[:20]), dict(name="b", tokens=b[:1])])
    logits = engine.step([dict(name="a", tokens=a[20:41], want=[0, 20]), dict(name="b", tokens=b[1:4], want=[2, 0])])
    want = [expected_output(s, 1)[0] for s in (a[:21], a[:41], b[:4], b[:2])]
    assert logits.argmax(-1).tolist() == want           # entry order, although the short portion runs first
    logits = engine.step([dict(name="b", tokens=b[4:], want=[40]), dict(name="a", tokens=a[41:42], want=[0])])
    assert logits.argmax(-1).tolist() == [expected_output(b, 1)[0], expected_output(a[:42], 1)[0]]
    assert engine.step([dict(name="a", tokens=a[42:43])]).shape == (0, 53)


def test_a_step_that_does_not_fit_changes_nothing(counting_engine):
    engine = counting_engine(max_tokens=64, max_sequences=2)
    engine.step([dict(name="a", tokens=[1] * 40)])
    free = engine.cache.free_pages
    for entries, error in (([dict(name="b", tokens=[1] * 17)], rlt.CacheFull), ([dict(name="b", tokens=[1]), dict(name="c", tokens=[1])], rlt.CacheFull),
                           ([dict(name="b", tokens=[99])], ValueError), ([dict(name="b", tokens=[1], want=[1])], ValueError),
                           ([dict(name="b", tokens=[])], ValueError), ([dict(name="b", tokens=[1]), dict(name="b", tokens=[1])], ValueError)):
        with pytest.raises(error):
            engine.step(entries)
        assert engine.cache.free_pages == free and "b" not in engine.cache and engine.cache.length("a") == 40


def test_generation_schedules_more_requests_than_fit(counting_engine):
    engine = counting_engine(max_tokens=128, max_sequences=2, max_step_tokens=24)
    prompts = [prompt(i, n, 53) for i, n in enumerate([70, 3, 20, 1, 33])]
    got = engine.generate(prompts, SamplingParams(max_tokens=9))
    assert got == [expected_output(p, 9) for p in prompts]
    assert engine.cache.free_pages == engine.cache.num_pages and engine.cache.free_slots == 2 and not engine.running


def test_decoding_goes_on_beside_a_long_prompt(counting_engine):
    engine = counting_engine(max_step_tokens=8)
    short, long = Request("short", [5, 6], SamplingParams(max_tokens=6)), Request("long", prompt(3, 40, 53), SamplingParams(max_tokens=1))
    engine.add_request(short)
    engine.run_step()
    engine.add_request(long)
    while not short.finished:
        before = len(short.generated_token_ids)
        engine.run_step()
        assert len(short.generated_token_ids) == before + 1
    assert not long.finished
    while not long.finished:
        engine.run_step()
    assert long.generated_token_ids == expected_output(long.prompt_token_ids, 1)


def test_requests_that_can_never_fit_are_refused(counting_engine):
    engine = counting_engine(max_tokens=64)
    with pytest.raises(ValueError, match="never fit"):
        engine.add_request(Request("x", [1] * 60, SamplingParams(max_tokens=6)))
    engine.add_request(Request("y", [1] * 60, SamplingParams(max_tokens=5)))


def test_trace_replay_writes_logits_and_gives_back(counting_engine, tmp_path):
    engine = counting_engine(max_tokens=64, max_sequences=4)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}, {"id": "b", "tokens": [4], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [5], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "c", "tokens": [9] * 48, "want": [47]}, {"id": "b", "tokens": [8], "want": [0]}], "end": ["b", "c"]}]
    answers = []
    trace.replay(engine, io.StringIO("\n".join(map(json.dumps, steps)) + "\n"), tmp_path, answers.append)
    assert answers == ["done 0", "done 1", "done 2"]
    assert sorted(p.name for p in tmp_path.iterdir()) == ["0.f32", "2.f32"]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, 53).argmax(-1).tolist()
    assert read(0) == [expected_output([1, 2, 3], 1)[0], expected_output([1], 1)[0]]
    assert read(2) == [expected_output([9] * 48, 1)[0], expected_output([4, 8], 1)[0]]
    assert engine.cache.free_pages == 4 and engine.cache.free_slots == 4


# ---- the plain functions themselves --------------------------------------------------------------
def test_plain_recurrence_against_its_closed_form():
    g = torch.Generator().manual_seed(0)
    n, size, p = 7, 3, 2
    x, b, c = torch.randn(n, 1, p, generator=g).double(), torch.randn(n, 1, size, generator=g).double(), torch.randn(n, 1, size, generator=g).double()
    dt_raw, a_log = torch.randn(n, 1, generator=g).double(), torch.tensor([0.3]).double()
    y, _ = plain.recurrence(x, b, c, dt_raw, torch.zeros(1).double(), a_log, torch.zeros(1).double())
    dt = torch.nn.functional.softplus(dt_raw[:, 0])
    for t in range(n):
        want = sum(torch.exp(-torch.exp(a_log[0]) * dt[s + 1:t + 1].sum()) * dt[s] * (c[t, 0] @ b[s, 0]) * x[s, 0] for s in range(t + 1))
        assert torch.allclose(y[t, 0], want)


def test_layers_the_package_builds_are_parsed_from_the_same_entries():
    config = rlt.HybridLMConfig.from_json(make_config([mamba_layer(2, 4, 6, 1), attention_layer(2, 1, 8, 4, temp=None, ff=None)]))
    assert config.layers[1].mixer.terms == rlt.ScoreTerms(8 ** -0.5, 0.0, 1, True) and config.layers[1].ff == 0
    assert config.layers[0].mixer.channels == 8 + 12
