"""Replaying a trace: given token ids through the engine's step function, one batch per step, logits to files.

Steps are read from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}

The entries of a step are one batch; a request is admitted at its first entry and keeps its pages and state until
a step lists it under "end".  A step that wants logits writes OUT/<step>.f32 — little-endian 32-bit floats,
[wanted, vocabulary], in the order of the entries and of "want" — and every step answers `done <step>`.
"""

from __future__ import annotations

import json
import sys
from pathlib import Path

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}
MAX_LIVE_REQUESTS = 4


def add_arguments(parser) -> None:
    parser.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    parser.add_argument("--dtype", choices=sorted(DTYPES), default="bfloat16")
    parser.add_argument("--out", required=True, help="folder for the logits files")
    parser.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at any time, in the cache pool")


def replay(engine, lines, out: Path, answer) -> None:
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [dict(name=e["id"], tokens=e["tokens"], want=e.get("want", [])) for e in step["entries"]]
        logits = engine.step(entries)
        if logits.shape[0]:
            data = logits.float().cpu().contiguous().numpy().astype("<f4", copy=False)
            (out / f"{step['step']}.f32").write_bytes(data.tobytes())
        for name in step.get("end", []):
            engine.release(name)
        answer(f"done {step['step']}")


def run(args) -> int:
    from . import build

    build.build()
    from .engine import Engine
    from .registry import load_model

    model = load_model(args.model, device="cuda", dtype=DTYPES[args.dtype])
    engine = Engine(model, max_tokens=args.max_tokens, max_sequences=MAX_LIVE_REQUESTS)
    replay(engine, sys.stdin, Path(args.out), lambda text: print(text, flush=True))
    return 0
