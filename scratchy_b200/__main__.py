"""Command line: `python -m scratchy_b200 generate --model DIR --tokens 1,2,3 --max-new-tokens 16` (greedy continuation of
token ids, one line per prompt), `python -m scratchy_b200 replay ...` (bin/trace_run)."""
from __future__ import annotations

import argparse
import sys

from . import trace


def generate(args) -> int:
    from .engine import Engine
    from .registry import load_model, prepare_library
    prepare_library(args.model)
    prompts = [[int(t) for t in p.split(",")] for p in args.tokens]
    model = load_model(args.model, "cuda", args.dtype, max_tokens=args.max_tokens, max_sequences=args.max_sequences)
    engine = Engine(model, step_tokens=args.step_tokens, max_batch=args.max_sequences)
    stop = [int(t) for t in args.stop.split(",")] if args.stop else []
    for out in engine.generate(prompts, args.max_new_tokens, stop):
        print(",".join(str(t) for t in out))
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="scratchy_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy continuation of token ids")
    g.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--tokens", action="append", required=True, help="a prompt as comma-separated token ids (repeat for a batch)")
    g.add_argument("--max-new-tokens", type=int, default=16)
    g.add_argument("--stop", default="", help="comma-separated token ids that end a continuation")
    g.add_argument("--max-tokens", type=int, default=8192)
    g.add_argument("--max-sequences", type=int, default=8)
    g.add_argument("--step-tokens", type=int, default=2048, help="most prompt tokens per step")
    r = sub.add_parser("replay", help="replay a trace of steps from standard input")
    trace.add_arguments(r)
    args = ap.parse_args(argv)
    return generate(args) if args.command == "generate" else trace.run(args)


if __name__ == "__main__":
    sys.exit(main())
