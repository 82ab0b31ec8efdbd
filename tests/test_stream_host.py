"""Host side of the decoder over hyper-connected streams, without a GPU: configuration, weights, cache, previous tokens and key
ranges of a step, and the plain functions that the GPU tests compare with."""

import json

import pytest
import torch

import plain_stream as plain
import vllm_rlt_b200 as rlt
from hybrid_cases import prompt, write_model
from stream_cases import CONFIGS, latent_layer, make_config, random_weights
from vllm_rlt_b200 import engine as engine_module
from vllm_rlt_b200 import registry, stream_lm
from vllm_rlt_b200.engine import KeyRanges
from vllm_rlt_b200.runner import SamplingParams


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configurations_parse_and_name_every_tensor(name):
    config = rlt.StreamLMConfig.from_json(CONFIGS[name])
    shapes = stream_lm.parameter_shapes(config)
    weights = random_weights(shapes, 0)
    model = rlt.StreamLM(config, weights, "cpu")
    for i, entry in enumerate(CONFIGS[name]["layers"]):
        layer = model.layers[i]
        assert len(layer.sublayers) == (2 if entry["mlp"] else 1)
        assert (f"l{i}.norm2" in shapes) == (f"l{i}.hc2.mix" in shapes) == bool(entry["mlp"])
        if entry["type"] == "latent_attention":
            assert torch.equal(layer.latent.w_down[layer.latent.kv_col:layer.latent.kv_col + layer.mixer.row], weights[f"l{i}.mix.dkv"])
            assert torch.equal(layer.latent.w_uk.reshape(-1, layer.mixer.kv_rank), weights[f"l{i}.mix.uk"])
        else:
            for at, n in ((layer.q_at, "q"), (layer.k_at, "k"), (layer.v_at, "v"), (layer.g_at, "g")):
                assert torch.equal(layer.w_in[at:at + weights[f"l{i}.mix.{n}"].shape[0]], weights[f"l{i}.mix.{n}"])
        if entry["mlp"] and entry["mlp"]["kind"] == "moe":
            assert torch.equal(layer.e_down[2], weights[f"l{i}.mlp.e2.down"])


def test_looped_layers_have_a_cache_for_every_pass():
    config = rlt.StreamLMConfig.from_json(CONFIGS["mixed"])
    assert config.runs == [0, 1, 2, 1, 2, 3]
    spec = rlt.StreamLM(config, random_weights(stream_lm.parameter_shapes(config), 0), "cpu").cache_spec()
    assert sorted(spec.layers) == [0, 2, 4] and spec.layers[4] == rlt.KVSpec(1, 36 + 8, 0)
    assert {k: v.shape for k, v in spec.states.items()} == {"r1.state": (5, 24, 40), "r3.state": (5, 24, 40), "r5.state": (2, 8, 16)}
    cache = rlt.SequenceCache(spec, max_tokens=64, max_sequences=2, device="cpu")
    assert spec.block == 64 and cache.key[0].shape == (4, 16, 1, 64) and not cache.value and cache.state["r5.state"].dtype == torch.float32


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0]["mixer"].update(sink=5), "unknown config keys"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(kind="chunk"), "unknown config keys"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "lacks"),
    (lambda c: c["layers"][0].update(type="attention"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=17), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=10), "top exceeds"),
    (lambda c: c["layers"][0]["mlp"].update(kind="shared"), "feed-forward"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][1]["mlp"].pop("limit"), "lacks"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["embedding"].update(trigram=True), "unknown config keys"),
    (lambda c: c.update(streams=0), "streams"),
])
def test_configurations_that_make_no_sense_are_refused(change, message):
    config = json.loads(json.dumps(CONFIGS["mixed"]))
    change(config)
    with pytest.raises(ValueError, match=message):
        rlt.StreamLMConfig.from_json(config)


def test_the_registry_loads_a_folder(tmp_path):
    config = rlt.StreamLMConfig.from_json(CONFIGS["odd"])
    weights = random_weights(stream_lm.parameter_shapes(config), 0)
    write_model(tmp_path, CONFIGS["odd"], weights)
    model = rlt.load_model(tmp_path, device="cpu", dtype=torch.float32)
    assert registry.resolve(CONFIGS["odd"]).model_class is rlt.StreamLM and model.config == config and model.embed.dtype == torch.float32
    del weights["l1.mlp.e1.up"]
    with pytest.raises(ValueError, match="lacks"):
        rlt.StreamLM(config, weights, "cpu")


class PairModel:
    """Next token = (5 * token + 3 * previous token + position) mod vocab, from what the engine hands over."""

    vocab_size, device, dtype = 47, torch.device("cpu"), torch.float32

    def cache_spec(self):
        return rlt.CacheSpec(layers={0: rlt.KVSpec(1, 1, 0)})

    def forward_step(self, batch, cache):
        for group in batch.groups:
            assert [list(p) for p in group.portions] == [[s, e - s] for s, e in zip(group.starts.tolist(), group.lengths.tolist())]
        return (5 * batch.tokens + 3 * batch.previous + batch.positions) % self.vocab_size

    def step_logits(self, hidden, rows=None):
        return torch.nn.functional.one_hot(hidden if rows is None else hidden[rows], self.vocab_size).float()


def test_the_previous_token_crosses_portions_and_ends_with_its_sequence(monkeypatch):
    monkeypatch.setattr(engine_module, "argmax_rows", lambda logits: logits.argmax(-1))
    engine = rlt.Engine(PairModel(), cuda_graphs=False, max_tokens=128, max_sequences=2, max_step_tokens=7)
    follow = lambda tokens: (5 * tokens[-1] + 3 * (tokens[-2] if len(tokens) > 1 else -1) + len(tokens) - 1) % 47
    prompts = [prompt(i, n, 47) for i, n in enumerate([30, 1, 2, 9, 20])]
    for p, out in zip(prompts, engine.generate(prompts, SamplingParams(max_tokens=6))):
        tokens = list(p)
        for token in out:
            assert token == follow(tokens)
            tokens.append(token)


def test_key_ranges_hold_what_the_rows_see():
    ranges = KeyRanges.of([(0, 5), (10, 3), (2, 1), (40, 20)], 4, torch.device("cpu"))
    assert ranges.first.tolist() == [0, 7, 0, 37] and ranges.cu.tolist() == [0, 5, 11, 14, 37] and ranges.rows == 37
    assert KeyRanges.of([(10, 300), (2, 20)], 4, torch.device("cpu")).tiles.tolist() == [
        [0, 256, 10, 0, 7, 0, 0, 0], [256, 44, 266, 0, 7, 0, 0, 0], [300, 20, 2, 303, 0, 0, 0, 0]]
    assert KeyRanges.of([(3, 5)], 0, torch.device("cpu")).first.tolist() == [0]
    assert KeyRanges.of([(3, 5)], 1, torch.device("cpu")).cu.tolist() == [0, 5]


# ---- the plain functions themselves --------------------------------------------------------------
def test_plain_rotation_depends_on_distance_only():
    g = torch.Generator().manual_seed(0)
    q, k = torch.randn(1, 10, generator=g).double(), torch.randn(1, 10, generator=g).double()
    at = lambda x, p: plain.rotate(x, torch.tensor([p]), 100.0, 8)
    assert torch.allclose((at(q, 17) * at(k, 5)).sum(), (at(q, 112) * at(k, 100)).sum())
    assert torch.equal(at(q, 9)[:, 8:], q[:, 8:]) and not torch.allclose(at(q, 9)[:, :8], q[:, :8])
    u, v = at(torch.tensor([[1.0, 0, 0, 0, 0, 0, 0, 0]]).double(), 1)[0, :2]
    assert torch.allclose(torch.stack([u, v]), torch.tensor([1.0, 1.0]).double().cos() * torch.tensor([1.0, 0]) + torch.tensor([0, 1.0]) * torch.tensor(1.0).double().sin())


def test_plain_window_and_decay_against_their_closed_forms():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(9, 2, 4, generator=g).double() for _ in range(3))
    out = plain.windowed_attention(q, k, v, 0.5, 3)
    for p in range(9):
        seen = [j for j in range(9) if 0 <= p - j < 3]
        w = torch.softmax((k[seen, 1] @ q[p, 1]) * 0.5, 0)
        assert torch.allclose(out[p, 1], w @ v[seen, 1])
    decay = torch.tensor([0.9, 0.2]).double()
    y, _ = plain.decayed_attention(q, k, v, decay)
    for t in range(9):
        assert torch.allclose(y[t, 0], sum(0.9 ** (t - s) * (k[s, 0] @ q[t, 0]) * v[s, 0] for s in range(t + 1)))


def test_one_stream_with_unit_coefficients_is_the_plain_residual():
    config = make_config([latent_layer(2, 8, 4, 8, 8, 8, 5)], streams=1, vocab=19, width=16, bigram=None)
    weights = random_weights(stream_lm.parameter_shapes(rlt.StreamLMConfig.from_json(config)), 3)
    for name in ("in", "out", "mix"):
        weights[f"l0.hc1.{name}"].fill_(1.0)
    model, layers, tokens = plain.PlainStream(config, weights), [], prompt(1, 7, 19)
    model(tokens, layers)
    x = model.embed(tokens)
    h = plain.rms_norm(x, model.w["l0.norm1"], 1e-5)
    assert torch.allclose(layers[0], x + model.latent("l0.mix.", config["layers"][0]["mixer"], h))


def test_steady_routes_choose_different_experts_without_close_calls():
    config = CONFIGS["wide"]
    weights = random_weights(stream_lm.parameter_shapes(rlt.StreamLMConfig.from_json(config)), 5, steady=True)
    seen, original = [], plain.route
    plain.route = lambda logits, correction, top: seen.append((logits, correction)) or original(logits, correction, top)
    try:
        plain.PlainStream(config, weights)(prompt(2, 40, config["vocab"]))
    finally:
        plain.route = original
    for logits, correction in seen:
        assert float(torch.sort(logits, 1).values.diff(dim=1).min()) > 0.02
        assert len(set(logits.argmax(1).tolist())) > 5
