"""The decoder over hyper-connected streams through the engine against the plain float64 model: whole prompts, portions, decoding,
mixed batches, pages and slots that change hands, windows, generation through the scheduler, the command line."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_stream as plain
import vllm_rlt_b200 as rlt
from hybrid_cases import prompt, write_model
from stream_cases import CONFIGS, latent_layer, make_config, moe, random_weights
from test_gpu_hybrid_model import check, feed, row_error
from vllm_rlt_b200 import stream_lm
from vllm_rlt_b200.runner import SamplingParams

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
DTYPES = [torch.float32, torch.bfloat16]
_MODELS: dict = {}
_PLAIN: dict = {}


def build(name, dtype, free=False):
    """Routers without close calls, or (`free`) any: a close call may fall the other way after the last bit of a sum."""
    if (name, dtype, free) not in _MODELS:
        config = rlt.StreamLMConfig.from_json(CONFIGS[name])
        weights = random_weights(stream_lm.parameter_shapes(config), 0, steady=not free)
        _MODELS[name, dtype, free] = (rlt.StreamLM(config, weights, "cuda", dtype), weights)
    return _MODELS[name, dtype, free]


def plain_run(name, dtype, tokens, rounded=0, free=False):
    """(logits, residual after every layer run) of the plain model."""
    key = (name, dtype, tuple(tokens), rounded, free)
    if key not in _PLAIN:
        layers = []
        _PLAIN[key] = plain.PlainStream(CONFIGS[name], build(name, dtype, free)[1], rounded)(tokens, layers), layers
    return _PLAIN[key]


def check_logits(got, name, tokens, dtype):
    """Logits at every position.  In bf16 a position may be off by three times what rounding the stored activations does to it."""
    want = plain_run(name, dtype, tokens)[0]
    if dtype == torch.float32:
        return check(got, want, dtype)
    rounding = torch.stack([row_error(plain_run(name, dtype, tokens, rounded=k)[0], want) for k in (1, 2, 3)]).amax(0)
    ratio = row_error(got, want) / torch.maximum(rounding, rounding.median())
    assert float(ratio.max()) < 3.0, (float(ratio.max()), int(ratio.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_residual_after_every_layer_run(name, dtype):
    free = dtype == torch.float32
    model, _ = build(name, dtype, free)
    tokens = prompt(4, 37, model.vocab_size)
    want, layers = plain_run(name, dtype, tokens, free=free)
    for cuts in ([37], [9, 20, 1]):
        engine = rlt.Engine(model, max_tokens=64, max_sequences=1, cuda_graphs=False)
        seen, original = {}, model.forward_step
        model.forward_step = lambda batch, cache: original(batch, cache, after_layer=lambda i, x: seen.setdefault(i, []).append(x.double().cpu()))
        try:
            logits = feed(engine, "s", tokens, cuts)
        finally:
            del model.forward_step
        check(logits, want, dtype)
        assert len(seen) == len(layers) == len(model.config.runs)
        for i, wanted in enumerate(layers):
            check(torch.cat(seen[i]), wanted, dtype)


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
    for tensor in [*engine.cache.key.values(), *engine.cache.state.values()]:
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
            check(feed(engine, "s", tokens[:n], [n]), plain_run(name, torch.float32, tokens)[0][:n], torch.float32)
            engine.release("s")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 16, 17, 64, 70])
def test_a_token_outside_the_window_changes_nothing(window, dtype):
    """One latent layer: logits at a position depend on the window's tokens and, through the bigram embedding of its first token, on
    one more; a change further back must not show at all, one inside must."""
    config = make_config([latent_layer(4, 64, 32, 64, 48, 64, window, base=50.0, mlp=moe(4, 4, 16))], streams=2, vocab=101, width=64)
    weights = random_weights(stream_lm.parameter_shapes(rlt.StreamLMConfig.from_json(config)), window)
    weights["l0.hc1.out"] *= 4                                       # the mixer's share of the streams stands out
    model = rlt.StreamLM(rlt.StreamLMConfig.from_json(config), weights, "cuda", dtype)
    tokens = prompt(window, 150, 101)
    for cuts in ([150], [145, 1], [40, 2]):
        def last(changed):
            engine = rlt.Engine(model, max_tokens=160, max_sequences=1)
            return feed(engine, "s", [(t + 1) % 101 if i == changed else t for i, t in enumerate(tokens)], cuts)[-1]
        base = last(None)
        assert torch.equal(last(149 - window - 1), base) and torch.equal(last(3), base)
        assert not torch.equal(last(149 - window + 1), base)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_follows_the_plain_model(name):
    model, _ = build(name, torch.float32)
    prompts = [prompt(20 + i, n, model.vocab_size) for i, n in enumerate([30, 4, 1, 50, 17])]
    engine = rlt.Engine(model, max_tokens=144, max_sequences=2, block=16, max_step_tokens=24)
    got = engine.generate(prompts, SamplingParams(max_tokens=12))
    for p, out in zip(prompts, got):
        assert plain_run(name, torch.float32, p + out[:-1])[0][len(p) - 1:].argmax(-1).tolist() == out
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
    want = plain_run("odd", torch.float32, tokens + generated[:-1])[0]
    assert generated == want[19:].argmax(-1).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": tokens[:12], "want": [0, 11]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": tokens[12:], "want": [7]}], "end": ["x"]}]
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"],
                         input="\n".join(map(json.dumps, steps)) + "\n", check=True, capture_output=True, text=True)
    assert [line for line in run.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1"]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, config["vocab"])
    check(torch.cat([read(0), read(1)]), want[[0, 11, 19]], torch.float32)
