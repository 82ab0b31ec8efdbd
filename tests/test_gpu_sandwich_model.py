"""The decoder with norms on both sides of its sublayers through the engine against the plain float64 model: whole prompts, portions,
decoding, mixed batches, pages and slots that change hands, windows, generation through the scheduler, the command line."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_sandwich as plain
import vllm_rlt_b200 as rlt
from hybrid_cases import prompt, write_model
from sandwich_cases import CONFIGS, latent_layer, make_config, random_weights, windowed_layer
from test_gpu_hybrid_model import check, feed, row_error
from vllm_rlt_b200 import sandwich_lm
from vllm_rlt_b200.runner import SamplingParams

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
DTYPES = [torch.float32, torch.bfloat16]
_MODELS: dict = {}
_PLAIN: dict = {}


def make(config, dtype, seed=0, change=None):
    parsed = rlt.SandwichLMConfig.from_json(config)
    weights = random_weights(sandwich_lm.parameter_shapes(parsed), seed)
    if change:
        change(weights)
    return rlt.SandwichLM(parsed, weights, "cuda", dtype), weights


def build(name, dtype):
    if (name, dtype) not in _MODELS:
        _MODELS[name, dtype] = make(CONFIGS[name], dtype)
    return _MODELS[name, dtype]


def plain_run(name, tokens, rounded=0):
    """(logits, residual after every layer) of the plain model."""
    key = (name, tuple(tokens), rounded)
    if key not in _PLAIN:
        layers = []
        _PLAIN[key] = plain.PlainSandwich(CONFIGS[name], build(name, torch.float32)[1], rounded)(tokens, layers), layers
    return _PLAIN[key]


def check_rows(got, want, rounded, dtype):
    """Rows of every position.  In bf16 a position may be off by three times what rounding the stored activations does to it."""
    if dtype == torch.float32:
        return check(got, want, dtype)
    rounding = torch.stack([row_error(other, want) for other in rounded]).amax(0)
    ratio = row_error(got, want) / torch.maximum(rounding, rounding.median())
    assert float(ratio.max()) < 3.0, (float(ratio.max()), int(ratio.argmax()))


def roundings(name, tokens, dtype):
    return [] if dtype == torch.float32 else [plain_run(name, tokens, rounded=k) for k in (1, 2, 3)]


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
@pytest.mark.parametrize("window,taps", [(1, 1), (1, 3), (16, 2), (17, 4), (64, 3), (70, 5)])
def test_a_token_outside_window_and_convolution_changes_nothing(window, taps, dtype):
    """One windowed layer: logits at a position depend on the window's tokens and, through the convolution of the first of them, on
    taps - 1 more; a change further back must not show at all, one at the edge must."""
    model, _ = make(make_config([windowed_layer(4, 2, 64, 64, taps, window)], vocab=101, width=64), dtype, window)
    tokens = prompt(window, 150, 101)
    for cuts in ([150], [145, 1], [40, 2]):
        def last(changed):
            engine = rlt.Engine(model, max_tokens=192, max_sequences=1)
            return feed(engine, "s", [(t + 1) % 101 if i == changed else t for i, t in enumerate(tokens)], cuts)[-1]
        base, edge = last(None), 149 - (window - 1) - (taps - 1)
        assert torch.equal(last(edge - 1), base) and torch.equal(last(3), base)
        assert not torch.equal(last(edge), base)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("second", [False, True])
def test_a_far_token_stands_out(second, dtype):
    """One latent layer whose queries and keys are steep: a position attends to one key in hundreds, the answer changes with it."""
    def steep(weights):
        weights["l0.mix.uq"] *= 4
        weights["l0.mix.uk"] *= 4
    config = make_config([latent_layer(2, 64, 16, 64, 48, 64, second=second, base=50.0)], vocab=101, width=64, mult=2.0)
    model, weights = make(config, dtype, 5, steep)
    reference = plain.PlainSandwich(config, weights)
    tokens = prompt(3, 330, 101)
    want = reference(tokens)
    rounded = [plain.PlainSandwich(config, weights, k)(tokens) for k in (1, 2, 3, 4)] if dtype == torch.bfloat16 else []
    for cuts in ([330], [300, 1], [100, 17, 2]):
        engine = rlt.Engine(model, max_tokens=384, max_sequences=1)
        check_rows(feed(engine, "s", tokens, cuts), want, rounded, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sinks_and_gates_change_the_answer(dtype):
    """The same weights without the sink, and with another gate, give other logits: neither is lost on any path."""
    config = make_config([latent_layer(4, 64, 16, 64, 48, 64, second=True)], vocab=101, width=64)
    tokens = prompt(7, 60, 101)
    def run(change, cuts):
        model, _ = make(config, dtype, 1, change)
        return feed(rlt.Engine(model, max_tokens=64, max_sequences=1), "s", tokens, cuts)
    def no_sink(w):
        w["l0.mix.sink"].fill_(-100.0)
    def other_gate(w):
        w["l0.mix.g"] *= -1
    for cuts in ([60], [1], [7]):
        base = run(None, cuts)
        for change in (no_sink, other_gate):
            assert float(row_error(run(change, cuts), base.double().cpu()).mean()) > 0.02


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
