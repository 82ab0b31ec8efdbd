"""The decoder that norms its sublayers' outputs through the engine against the plain float64 model: whole prompts, portions, decoding,
mixed batches, pages and slots that change hands, windows and kept tokens, shared weights, generation through the scheduler, the command line."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_postnorm as plain
import vllm_rlt_b200 as rlt
from hybrid_cases import prompt, write_model
from postnorm_cases import CONFIGS, again, attention_layer, delta_layer, make_config, rank_of, random_weights, retention_layer
from test_gpu_hybrid_model import check, feed, row_error
from vllm_rlt_b200 import postnorm_lm
from vllm_rlt_b200.runner import SamplingParams

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
DTYPES = [torch.float32, torch.bfloat16]
_MODELS: dict = {}
_PLAIN: dict = {}


def make(config, dtype, seed=0, change=None, ranks=lambda name: 8):
    parsed = rlt.PostNormLMConfig.from_json(config)
    weights = random_weights(postnorm_lm.parameter_shapes(parsed, ranks), seed)
    if change:
        change(weights)
    return rlt.PostNormLM(parsed, weights, "cuda", dtype), weights


def build(name, dtype):
    if (name, dtype) not in _MODELS:
        _MODELS[name, dtype] = make(CONFIGS[name], dtype, ranks=rank_of(name))
    return _MODELS[name, dtype]


def plain_run(name, tokens, rounded=0):
    """(logits, residual after every layer) of the plain model."""
    key = (name, tuple(tokens), rounded)
    if key not in _PLAIN:
        layers = []
        _PLAIN[key] = plain.PlainPostNorm(CONFIGS[name], build(name, torch.float32)[1], rounded)(tokens, layers), layers
    return _PLAIN[key]


def check_rows(got, want, rounded, dtype):
    """Rows of every position.  In bf16 a position may be off by three times what rounding the stored activations does to it."""
    if dtype == torch.float32:
        return check(got, want, dtype)
    rounding = torch.stack([row_error(other, want) for other in rounded]).amax(0)
    ratio = row_error(got, want) / torch.maximum(rounding, rounding.median())
    assert float(ratio.max()) < 3.0, (float(ratio.max()), int(ratio.argmax()))


def roundings(name, tokens, dtype):
    return [] if dtype == torch.float32 else [plain_run(name, tokens, rounded=k) for k in range(1, 6)]


def check_logits(got, name, tokens, dtype):
    check_rows(got, plain_run(name, tokens)[0], [r[0] for r in roundings(name, tokens, dtype)], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_residual_after_every_layer(name, dtype):
    model, _ = build(name, dtype)
    tokens = prompt(4, 37, model.vocab_size)
    want, layers = plain_run(name, tokens)
    for cuts in ([37], [9, 20, 1]):
        engine = rlt.Engine(model, max_tokens=64, max_sequences=1, cuda_graphs=False)
        seen, original = {}, model.forward_step
        model.forward_step = lambda batch, cache: original(batch, cache, after_layer=lambda i, x: seen.setdefault(i, []).append(x.double().cpu()))
        try:
            check_logits(feed(engine, "s", tokens, cuts), name, tokens, dtype)
        finally:
            del model.forward_step
        assert len(seen) == len(layers) == len(model.config.layers)
        for i, wanted in enumerate(layers):
            check_rows(torch.cat(seen[i]), wanted, [r[1][i] for r in roundings(name, tokens, dtype)], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("block", [16, 64])
@pytest.mark.parametrize("cuts", [[200], [1], [2], [3, 17, 40, 5, 16, 2], [64, 1], [33], [150, 20, 2]], ids=str)
def test_logits_do_not_depend_on_the_cut(name, dtype, cuts, block):
    model, _ = build(name, dtype)
    tokens = prompt(1, 200, model.vocab_size)
    engine = rlt.Engine(model, max_tokens=256, max_sequences=2, block=block)
    check_logits(feed(engine, "s", tokens, cuts), name, tokens, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_requests_in_mixed_batches_over_reused_pages(name, graphs, dtype):
    """Six requests over room for three: portions of some beside single tokens of others, in a pool that is handed on again and
    again; requests pause and go on."""
    model, _ = build(name, dtype)
    engine = rlt.Engine(model, max_tokens=160, max_sequences=3, block=16, cuda_graphs=graphs)
    lengths = [70, 1, 33, 5, 48, 90]
    texts = [prompt(10 + i, n, model.vocab_size) for i, n in enumerate(lengths)]
    portions = [1, 7, 20, 1, 1, 16, 2, 40, 1, 3, 17, 1]
    waiting, live, at, got, turn, users = list(range(6)), [], {}, {i: [] for i in range(6)}, 0, {}
    while waiting or live:
        while waiting and len(live) < 3 and sum(-(-lengths[i] // 16) for i in live + waiting[:1]) <= 10:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        entries = []
        for k, i in enumerate(live):
            if (turn + k) % 5 == 4 and len(live) > 1:
                continue                                              # left out of this step
            n = portions[(turn + 2 * k) % len(portions)] if turn % 4 != 3 else 1      # every fourth step is all decoding
            entries.append(rlt.StepEntry(i, texts[i][at[i]:at[i] + n], list(range(min(n, lengths[i] - at[i])))))
        turn += 1
        if not entries:
            continue
        rows, first = engine.step(entries), 0
        for e in entries:
            got[e.name].append(rows[first:first + len(e.tokens)])
            first += len(e.tokens)
            at[e.name] += len(e.tokens)
            for page in engine.cache.pages(e.name):
                users.setdefault(page, set()).add(e.name)
            if at[e.name] == lengths[e.name]:
                engine.release(e.name)
                live.remove(e.name)
    assert max(len(u) for u in users.values()) > 1
    for i in range(6):
        check_logits(torch.cat(got[i]), name, texts[i], dtype)
    assert engine.cache.free_pages == engine.cache.num_pages and engine.cache.free_slots == 3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_stale_pages_and_slots_never_show(name, dtype):
    """Everything a new sequence could wrongly read is poisoned before it starts."""
    model, _ = build(name, dtype)
    engine = rlt.Engine(model, max_tokens=64, max_sequences=1)
    for tensor in [*engine.cache.key.values(), *engine.cache.value.values(), *engine.cache.state.values()]:
        tensor.fill_(float("nan"))
    for cuts in ([2, 1], [20, 1], [1], [30]):
        tokens = prompt(sum(cuts), 30, model.vocab_size)
        check_logits(feed(engine, "s", tokens, cuts), name, tokens, dtype)
        engine.release("s")
        for tensor in engine.cache.state.values():
            tensor.fill_(float("nan"))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """Hundreds of decoded tokens behind a short prompt: across pages and past every window."""
    model, _ = build("mixed", dtype)
    tokens = prompt(8, 420, model.vocab_size)
    engine = rlt.Engine(model, max_tokens=448, max_sequences=1)
    check_logits(feed(engine, "s", tokens, [9, 1]), "mixed", tokens, dtype)
    engine.release("s")
    check_logits(feed(engine, "s", tokens, [420]), "mixed", tokens, dtype)


def test_first_tokens_of_a_sequence():
    for name in sorted(CONFIGS):
        model, _ = build(name, torch.float32)
        engine = rlt.Engine(model, max_tokens=16, max_sequences=1)
        tokens = prompt(6, 6, model.vocab_size)
        for n in range(1, 7):
            check(feed(engine, "s", tokens[:n], [n]), plain_run(name, tokens)[0][:n], torch.float32)
            engine.release("s")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep", [(1, 0), (1, 1), (16, 3), (17, 16), (64, 4), (70, 65)])
def test_a_token_outside_the_window_and_behind_the_kept_ones_changes_nothing(window, keep, dtype):
    model, _ = make(make_config([attention_layer(4, 2, 64, 64, window, keep)], vocab=101, width=64), dtype, window)
    tokens = prompt(window, 150, 101)
    for cuts in ([150], [145, 1], [40, 2]):
        def last(changed):
            engine = rlt.Engine(model, max_tokens=192, max_sequences=1)
            return feed(engine, "s", [(t + 1) % 101 if i == changed else t for i, t in enumerate(tokens)], cuts)[-1]
        base, edge = last(None), 149 - (window - 1)
        assert torch.equal(last(edge - 1), base) and torch.equal(last(keep), base)
        assert not torch.equal(last(edge), base)
        if keep:
            assert not torch.equal(last(keep - 1), base) and not torch.equal(last(0), base)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [delta_layer(2, 2, 64, 64, 4), retention_layer(2, 64, 64, decay=[1.0, 0.9999])], ids=["delta", "retention"])
def test_a_far_token_is_remembered(layer, dtype):
    """Hardly any decay: the answer hundreds of tokens later still depends on the first token, however the text is cut."""
    def slow(weights):
        for name in weights:
            if name.endswith("dt_bias"):
                weights[name].fill_(-14.0)
    config = make_config([layer], vocab=101, width=64)
    model, weights = make(config, dtype, 5, slow)
    tokens = prompt(3, 330, 101)
    want = plain.PlainPostNorm(config, weights)(tokens)
    rounded = [plain.PlainPostNorm(config, weights, k)(tokens) for k in (1, 2, 3, 4)] if dtype == torch.bfloat16 else []
    for cuts in ([330], [300, 1], [100, 17, 2]):
        engine = rlt.Engine(model, max_tokens=384, max_sequences=1)
        got = feed(engine, "s", tokens, cuts)
        check_rows(got, want, rounded, dtype)
        engine.release("s")
        other = feed(engine, "s", [(tokens[0] + 1) % 101, *tokens[1:]], cuts)
        assert not torch.equal(other[-1], got[-1])


@pytest.mark.parametrize("dtype", DTYPES)
def test_layers_that_share_weights_keep_a_cache_each(dtype):
    """The same layer three times is the model with three copies of its weights."""
    layers = [delta_layer(2, 1, 16, 24, 3, mlp={"kind": "dense", "ff": 40}), attention_layer(4, 2, 16, 24, 9, 2), retention_layer(2, 16, 8)]
    shared = make_config([*layers, again(layers, 0), again(layers, 1), again(layers, 2), {**again(layers, 1), "weights_of": 4}], vocab=61, width=32)
    copies = make_config([*layers, *layers, layers[1]], vocab=61, width=32)
    model, weights = make(shared, dtype, 2)
    source = {3: 0, 4: 1, 5: 2, 6: 1}
    full = {n: t for n, t in weights.items()}
    for i, j in source.items():
        full.update({f"l{i}." + n.split(".", 1)[1]: t for n, t in weights.items() if n.startswith(f"l{j}.")})
    other = rlt.PostNormLM(rlt.PostNormLMConfig.from_json(copies), full, "cuda", dtype)
    tokens = prompt(9, 70, 61)
    for cuts in ([70], [20, 1]):
        a, b = (feed(rlt.Engine(m, max_tokens=128, max_sequences=1), "s", tokens, cuts) for m in (model, other))
        assert torch.equal(a, b)
    assert len(model.cache_spec().layers) == 3 and len(model.cache_spec().states) == 6


@pytest.mark.parametrize("dtype", DTYPES)
def test_talking_and_temperatures_change_the_answer(dtype):
    config = make_config([attention_layer(4, 2, 64, 64, 30, 2)], vocab=101, width=64)
    tokens = prompt(7, 60, 101)
    def run(change, cuts):
        model, _ = make(config, dtype, 1, change)
        return feed(rlt.Engine(model, max_tokens=64, max_sequences=1), "s", tokens, cuts)
    def silent(w):
        w["l0.mix.talk"].copy_(torch.eye(4))
    def transposed(w):
        w["l0.mix.talk"].copy_(w["l0.mix.talk"].t().clone())
    def even(w):
        w["l0.mix.temp"].fill_(1.0)
    for cuts in ([60], [1], [7]):
        base = run(None, cuts)
        for change in (silent, transposed, even):
            assert float(row_error(run(change, cuts), base.double().cpu()).mean()) > 0.01


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_follows_the_plain_model(name):
    model, _ = build(name, torch.float32)
    prompts = [prompt(20 + i, n, model.vocab_size) for i, n in enumerate([30, 4, 1, 50, 17])]
    engine = rlt.Engine(model, max_tokens=144, max_sequences=2, block=16, max_step_tokens=24)
    got = engine.generate(prompts, SamplingParams(max_tokens=12))
    for p, out in zip(prompts, got):
        assert plain_run(name, p + out[:-1])[0][len(p) - 1:].argmax(-1).tolist() == out
    eager = rlt.Engine(model, max_tokens=512, max_sequences=5, cuda_graphs=False)
    assert eager.generate(prompts, SamplingParams(max_tokens=12)) == got


def test_sampled_generation_is_reproducible_and_independent_of_the_batch():
    model, _ = build("mixed", torch.float32)
    prompts = [prompt(40 + i, 8 + i, model.vocab_size) for i in range(4)]
    params = [SamplingParams(max_tokens=10, temperature=0.9, top_k=20, top_p=0.95, seed=100 + i) for i in range(4)]
    engine = rlt.Engine(model, max_tokens=256, max_sequences=4)
    got = engine.generate(prompts, params)
    assert got == engine.generate(prompts, params)
    for p, s, out in zip(prompts, params, got):
        assert engine.generate([p], [s]) == [out]


def test_command_line_and_trace_agree_with_the_engine(tmp_path):
    config, folder = CONFIGS["odd"], tmp_path / "model"
    write_model(folder, config, build("odd", torch.float32)[1])
    tokens = prompt(3, 20, config["vocab"])
    out = subprocess.run([sys.executable, "-m", "vllm_rlt_b200", "generate", "--model", str(folder), "--dtype", "float32", "--prompt",
                          ",".join(map(str, tokens)), "--max-tokens", "5"], cwd=ROOT, check=True, capture_output=True, text=True).stdout
    generated = json.loads(out.strip().splitlines()[-1])
    want = plain_run("odd", tokens + generated[:-1])[0]
    assert generated == want[19:].argmax(-1).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": tokens[:12], "want": [0, 11]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": tokens[12:], "want": [7]}], "end": ["x"]}]
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"],
                         input="\n".join(map(json.dumps, steps)) + "\n", check=True, capture_output=True, text=True)
    assert [line for line in run.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1"]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, config["vocab"])
    check(torch.cat([read(0), read(1)]), want[[0, 11, 19]], torch.float32)
