"""The hybrid decoder through the engine against the plain float64 model: whole prompts, portions, decoding, mixed
batches, pages and slots that change hands, generation through the scheduler, the command line."""

import io
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_hybrid as plain
import vllm_rlt_b200 as rlt
from hybrid_cases import CONFIGS, prompt, random_weights, write_model
from vllm_rlt_b200 import hybrid_lm, trace
from vllm_rlt_b200.runner import SamplingParams

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
_MODELS: dict = {}
_LOGITS: dict = {}


def build(name, dtype, seed=0):
    if (name, dtype, seed) not in _MODELS:
        config = rlt.HybridLMConfig.from_json(CONFIGS[name])
        weights = random_weights(hybrid_lm.parameter_shapes(config), seed)
        _MODELS[name, dtype, seed] = (rlt.HybridLM(config, weights, "cuda", dtype), plain.PlainHybrid(config, weights))
    return _MODELS[name, dtype, seed]


def plain_logits(name, tokens, seed=0):
    key = (name, tuple(tokens), seed)
    if key not in _LOGITS:
        _LOGITS[key] = build(name, torch.float32, seed)[1](tokens)
    return _LOGITS[key]


def row_error(got, want):
    """Root mean square of the difference over a row, against that of all rows."""
    got, want = got.double().cpu(), want.double()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


def check(got, want, dtype):
    error = row_error(got, want)
    assert float(error.max()) < {torch.float32: 3e-5, torch.bfloat16: 4e-2}[dtype], float(error.max())


def check_logits(got, name, tokens, dtype):
    """Logits at every position of a sequence.  In bf16 a position may be off by three times what rounding the stored
    activations of the plain model does to it (some positions amplify it: norm groups of a few nearly cancelling values)."""
    want = plain_logits(name, tokens)
    if dtype == torch.float32:
        return check(got, want, dtype)
    key = (name, tuple(tokens), "rounded")
    if key not in _LOGITS:
        config, weights = build(name, dtype)[0].config, build(name, torch.float32)[1].w
        _LOGITS[key] = row_error(plain.PlainHybrid(config, weights, rounded=True)(tokens), want)
    rounding = _LOGITS[key]
    ratio = row_error(got, want) / torch.maximum(rounding, rounding.median())
    assert float(ratio.max()) < 3.0, (float(ratio.max()), int(ratio.argmax()))


def feed(engine, name, tokens, cuts):
    """The sequence's logits at every position, portion by portion (the last cut repeats)."""
    rows, at = [], 0
    cuts = list(cuts)
    while at < len(tokens):
        n = cuts.pop(0) if len(cuts) > 1 else cuts[0]
        portion = tokens[at:at + n]
        rows.append(engine.step([rlt.StepEntry(name, portion, list(range(len(portion))))]))
        at += n
    return torch.cat(rows)


DTYPES = [torch.float32, torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_residual_after_every_layer(name, dtype):
    model, reference = build(name, dtype)
    tokens = prompt(4, 37, model.vocab_size)
    engine = rlt.Engine(model, max_tokens=64, max_sequences=1, cuda_graphs=False)
    seen, original = [], model.forward_step
    model.forward_step = lambda batch, cache: original(batch, cache, after_layer=lambda i, x: seen.append(x.double().cpu()))
    try:
        logits = engine.step([rlt.StepEntry("s", tokens, list(range(37)))])
    finally:
        del model.forward_step
    wanted = []
    check(logits, reference(tokens, wanted), dtype)
    assert len(seen) == len(wanted) == len(model.config.layers)
    for got, want in zip(seen, wanted):
        check(got, want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("cuts", [[97], [1], [2], [3, 17, 40, 5, 16, 2], [64, 1], [33]], ids=str)
def test_logits_do_not_depend_on_the_cut(name, dtype, cuts):
    model, _ = build(name, dtype)
    tokens = prompt(1, 97, model.vocab_size)
    engine = rlt.Engine(model, max_tokens=112, max_sequences=2)
    check_logits(feed(engine, "s", tokens, cuts), name, tokens, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_requests_in_mixed_batches_over_reused_pages(name, graphs, dtype):
    """Six requests over room for three: portions of some beside single tokens of others, in a pool that is handed on
    again and again; requests pause and go on."""
    model, _ = build(name, dtype)
    engine = rlt.Engine(model, max_tokens=160, max_sequences=3, cuda_graphs=graphs)
    lengths = [70, 1, 33, 5, 48, 90]
    texts = [prompt(10 + i, n, model.vocab_size) for i, n in enumerate(lengths)]
    portions = [1, 7, 20, 1, 1, 16, 2, 40, 1, 3, 17, 1]
    waiting, live, at, got, turn, pages_seen = list(range(6)), [], {}, {i: [] for i in range(6)}, 0, {}
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
                pages_seen.setdefault(page, set()).add(e.name)
            if at[e.name] == lengths[e.name]:
                engine.release(e.name)
                live.remove(e.name)
    assert max(len(users) for users in pages_seen.values()) > 1
    for i in range(6):
        check_logits(torch.cat(got[i]), name, texts[i], dtype)
    assert engine.cache.free_pages == engine.cache.num_pages and engine.cache.free_slots == 3


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_stale_pages_and_slots_never_show(name):
    """Everything a new sequence could wrongly read is poisoned before it starts."""
    model, _ = build(name, torch.float32)
    engine = rlt.Engine(model, max_tokens=64, max_sequences=1)
    for tensor in [*engine.cache.key.values(), *engine.cache.value.values(), *engine.cache.state.values()]:
        tensor.fill_(float("nan"))
    for cuts in ([2, 1], [20, 1], [1]):
        tokens = prompt(sum(cuts), 30, model.vocab_size)
        check(feed(engine, "s", tokens, cuts), plain_logits(name, tokens), torch.float32)
        engine.release("s")
        for tensor in engine.cache.state.values():
            tensor.fill_(float("nan"))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """Hundreds of decoded tokens behind a short prompt: across pages, temperature steps and attention chunks."""
    model, _ = build("wide", dtype)
    tokens = prompt(8, 620, model.vocab_size)
    engine = rlt.Engine(model, max_tokens=624, max_sequences=1)
    got = feed(engine, "s", tokens, [9, 1])
    check_logits(got, "wide", tokens, dtype)
    engine.release("s")
    check_logits(feed(engine, "s", tokens, [620]), "wide", tokens, dtype)


def test_first_tokens_of_a_sequence():
    for name in sorted(CONFIGS):
        model, _ = build(name, torch.float32)
        engine = rlt.Engine(model, max_tokens=16, max_sequences=1)
        tokens = prompt(6, 6, model.vocab_size)
        for n in range(1, 7):
            check(feed(engine, "s", tokens[:n], [n]), plain_logits(name, tokens)[:n], torch.float32)
            engine.release("s")


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_follows_the_plain_model(name):
    model, reference = build(name, torch.float32)
    prompts = [prompt(20 + i, n, model.vocab_size) for i, n in enumerate([30, 4, 1, 50, 17])]
    engine = rlt.Engine(model, max_tokens=144, max_sequences=2, max_step_tokens=24)
    got = engine.generate(prompts, SamplingParams(max_tokens=12))
    for p, out in zip(prompts, got):
        logits = reference(p + out[:-1])[len(p) - 1:]
        assert logits.argmax(-1).tolist() == out
    eager = rlt.Engine(model, max_tokens=512, max_sequences=5, cuda_graphs=False)
    assert eager.generate(prompts, SamplingParams(max_tokens=12)) == got


def test_sampled_generation_is_reproducible_and_independent_of_the_batch():
    model, _ = build("odd", torch.float32)
    prompts = [prompt(40 + i, 8 + i, model.vocab_size) for i in range(4)]
    params = [SamplingParams(max_tokens=10, temperature=0.9, top_k=20, top_p=0.95, seed=100 + i) for i in range(4)]
    engine = rlt.Engine(model, max_tokens=256, max_sequences=4)
    got = engine.generate(prompts, params)
    assert got == engine.generate(prompts, params)
    for p, s, out in zip(prompts, params, got):
        assert engine.generate([p], [s]) == [out]
    assert engine.generate(prompts, [SamplingParams(10, 0.9, seed=7 + i) for i in range(4)]) != got
    cold = engine.generate(prompts, [SamplingParams(10, 1e-4, seed=i) for i in range(4)])
    assert cold == engine.generate(prompts, SamplingParams(max_tokens=10))


def test_command_line_and_trace_agree_with_the_engine(tmp_path):
    config, folder = CONFIGS["odd"], tmp_path / "model"
    weights = random_weights(hybrid_lm.parameter_shapes(rlt.HybridLMConfig.from_json(config)), 0)
    write_model(folder, config, weights)
    tokens = prompt(3, 20, config["vocab"])
    out = subprocess.run([sys.executable, "-m", "vllm_rlt_b200", "generate", "--model", str(folder), "--dtype", "float32", "--prompt",
                          ",".join(map(str, tokens)), "--max-tokens", "5"], cwd=ROOT, check=True, capture_output=True, text=True).stdout
    generated = json.loads(out.strip().splitlines()[-1])
    want = plain_logits("odd", tokens + generated[:-1])
    assert generated == want[19:].argmax(-1).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": tokens[:12], "want": [0, 11]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": tokens[12:], "want": [7]}], "end": ["x"]}]
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"],
                         input="\n".join(map(json.dumps, steps)) + "\n", check=True, capture_output=True, text=True)
    assert [line for line in run.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1"]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, config["vocab"])
    check(torch.cat([read(0), read(1)]), want[[0, 11, 19]], torch.float32)


def test_the_engine_serves_the_looped_model_too():
    """The framework's other family through the same engine: the tokens of its own native decoding."""
    config = rlt.LoopedLMConfig(vocab_size=97, hidden_size=64, intermediate_size=96, num_hidden_layers=2, num_attention_heads=4,
                                num_key_value_heads=2, head_dim=16, total_ut_steps=3, initializer_range=0.2)
    model = rlt.LoopedLM(config, rlt.seeded_state_dict(config, 3), "cuda", torch.float32)
    prompts = [prompt(60 + i, n, 97) for i, n in enumerate([21, 3, 40])]
    want = rlt.SelfSpeculativeDecoder(model).generate_native(prompts, 8)
    engine = rlt.Engine(model, max_tokens=128, max_sequences=2, max_step_tokens=20)
    assert engine.generate(prompts, SamplingParams(max_tokens=8)) == want
    sink = []
    trace.replay(rlt.Engine(model, max_tokens=64, max_sequences=4), io.StringIO(json.dumps({"step": 0, "entries": [{"id": "q", "tokens": prompts[1]}]})),
                 None, sink.append)
    assert sink == ["done 0"]
