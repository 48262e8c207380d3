"""Command line of the framework.

    bin/b200_serve models                            architectures the registry knows
    bin/b200_serve generate --model DIR --prompt 1,2,3 [--prompt ...] --new-tokens N
    bin/trace_run --model DIR --dtype bfloat16 --out DIR --max-tokens N < steps.jsonl
"""

from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import List, Optional

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32, "float16": torch.float16}
TRACE_SLOTS = 8  # sequences a replayed trace may hold at once


def ensure_built() -> None:
    """Compiles the kernel library if it is missing or older than its sources."""

    from . import build

    build.build()


def _trace(args: argparse.Namespace) -> int:
    from .registry import load_model
    from .trace import replay

    out = Path(args.out)
    out.mkdir(parents=True, exist_ok=True)
    engine = load_model(args.model, dtype=DTYPES[args.dtype], batch=TRACE_SLOTS, capacity=args.max_tokens)
    replay(engine, sys.stdin, out, sys.stdout)
    return 0


def _generate(args: argparse.Namespace) -> int:
    from .registry import entry_of, load_model
    from .scheduler import RequestScheduler

    prompts = [[int(t) for t in text.split(",")] for text in args.prompt]
    longest = max(map(len, prompts)) + args.new_tokens
    portions = entry_of(json.loads((Path(args.model) / "config.json").read_text())).portions
    engine = load_model(args.model, dtype=DTYPES[args.dtype], batch=min(len(prompts), args.max_batch) if portions else len(prompts),
                        capacity=longest)
    if portions:
        scheduler = RequestScheduler(engine, max_portion=args.max_portion)
        requests = [scheduler.submit(prompt, args.new_tokens) for prompt in prompts]
        scheduler.run()
        outputs = [request.output for request in requests]
    else:
        if len({len(p) for p in prompts}) != 1:
            raise SystemExit("this engine serves prompts of one length per batch")
        outputs = engine.generate(torch.tensor(prompts), args.new_tokens - 1).tolist()
    for prompt, output in zip(prompts, outputs):
        print(json.dumps({"prompt": prompt, "output": output}))
    return 0


def _models(args: argparse.Namespace) -> int:
    from .registry import architectures

    print("\n".join(architectures()))
    return 0


def trace_main(argv: Optional[List[str]] = None) -> int:
    parser = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace and write its logits.")
    parser.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    parser.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    parser.add_argument("--out", required=True, help="folder for the logits")
    parser.add_argument("--max-tokens", type=int, required=True, help="most tokens a live sequence holds")
    args = parser.parse_args(argv)
    ensure_built()
    return _trace(args)


def main(argv: Optional[List[str]] = None) -> int:
    parser = argparse.ArgumentParser(prog="b200_serve", description="Serve a model of the registry.")
    commands = parser.add_subparsers(dest="command", required=True)
    commands.add_parser("models", help="list the registry").set_defaults(run=_models)
    generate = commands.add_parser("generate", help="greedy generation from token ids")
    generate.add_argument("--model", required=True)
    generate.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    generate.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; repeatable")
    generate.add_argument("--new-tokens", type=int, default=16)
    generate.add_argument("--max-batch", type=int, default=64)
    generate.add_argument("--max-portion", type=int, default=2048, help="prompt tokens between two decode steps")
    generate.set_defaults(run=_generate)
    args = parser.parse_args(argv)
    if args.command != "models":
        ensure_built()
    return args.run(args)
