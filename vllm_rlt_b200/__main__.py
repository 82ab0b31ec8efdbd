"""Command line of the framework.

    python -m vllm_rlt_b200 models
    python -m vllm_rlt_b200 generate --model DIR --prompt 5,17,3 [--prompt ...] [--max-tokens N] [--temperature T] ...
    python -m vllm_rlt_b200 trace --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Prompts and outputs are token ids (the framework has no tokenizer); a model folder holds config.json, whose
architecture selects the model class, and safetensors weights.
"""

from __future__ import annotations

import argparse
import json
import sys


def _generate(args) -> int:
    import torch

    from . import build

    build.build()
    from .engine import Engine
    from .registry import load_model
    from .runner import SamplingParams

    prompts = [[int(t) for t in text.replace(",", " ").split()] for text in args.prompt]
    if args.prompts_file:
        with open(args.prompts_file) as f:
            prompts += [json.loads(line) for line in f if line.strip()]
    if not prompts or not all(prompts):
        raise SystemExit("generate: give at least one nonempty --prompt or a --prompts-file")
    model = load_model(args.model, device="cuda", dtype={"bfloat16": torch.bfloat16, "float32": torch.float32}[args.dtype])
    page = model.cache_spec().block
    pool = args.pool_tokens or sum(-(-(len(p) + args.max_tokens) // page) * page for p in prompts)
    engine = Engine(model, max_tokens=pool, max_sequences=min(args.max_sequences, len(prompts)),
                    max_step_tokens=args.max_step_tokens, cuda_graphs=not args.eager)
    params = SamplingParams(args.max_tokens, args.temperature, args.top_p, args.top_k, args.seed)
    for tokens in engine.generate(prompts, params):
        print(json.dumps(tokens), flush=True)
    return 0


def _models(args) -> int:
    from .registry import registered_architectures

    print("\n".join(registered_architectures()))
    return 0


def main(argv=None) -> int:
    from . import trace

    parser = argparse.ArgumentParser(prog="python -m vllm_rlt_b200", description="B200-native serving of the registered models")
    commands = parser.add_subparsers(dest="command", required=True)
    commands.add_parser("models", help="list the registered architectures").set_defaults(run=_models)
    g = commands.add_parser("generate", help="generate from token id prompts; one JSON list of token ids per prompt")
    g.add_argument("--model", required=True)
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--prompt", action="append", default=[], help="token ids, separated by commas or spaces (repeatable)")
    g.add_argument("--prompts-file", help="one JSON list of token ids per line")
    g.add_argument("--max-tokens", type=int, default=16)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=-1)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--max-sequences", type=int, default=64, help="requests that run together")
    g.add_argument("--max-step-tokens", type=int, default=8192, help="rows of one step")
    g.add_argument("--pool-tokens", type=int, default=None, help="cache pool size (default: all prompts and outputs)")
    g.add_argument("--eager", action="store_true", help="launch decode steps kernel by kernel instead of from CUDA graphs")
    g.set_defaults(run=_generate)
    t = commands.add_parser("trace", help="replay given token ids step by step and write logits")
    trace.add_arguments(t)
    t.set_defaults(run=trace.run)
    args = parser.parse_args(argv)
    return args.run(args)


if __name__ == "__main__":
    sys.exit(main())
