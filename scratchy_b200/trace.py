"""Replays a trace through the engine: steps of given token ids from standard input, logits to files.

A line of input is one step, `{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}`: the
next tokens of each request, the places among them whose logits are wanted, and the requests that are over after the
step.  Logits go to `<out>/<n>.f32` (little-endian f32, [wanted, vocab]); `done <n>` follows on standard output."""
from __future__ import annotations

import argparse
import json
import os
import sys

from . import _lib

REFUSED = 3          # exit code: no model of this architecture runs in the requested number format


def add_arguments(ap: argparse.ArgumentParser) -> None:
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits of each step")
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-sequences", type=int, default=16, help="most requests alive at any time")


def run(args, lines=None, out=None) -> int:
    lines, out = lines if lines is not None else sys.stdin, out if out is not None else sys.stdout
    from .engine import Engine
    from .registry import load_model, prepare_library
    try:
        prepare_library(args.model)
        model = load_model(args.model, "cuda", args.dtype, max_tokens=args.max_tokens, max_sequences=args.max_sequences)
    except _lib.ScratchyCudaError as e:
        if e.status == -4:                       # SCR_E_DTYPE
            print(e, file=sys.stderr)
            return REFUSED
        raise
    engine = Engine(model)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]]
        # logits are returned in ascending order of place; hand them out in the order asked for
        ordered = [(name, tokens, sorted(set(want))) for name, tokens, want in entries]
        logits = engine.run_step(ordered, step.get("end", []))
        if logits is not None:
            rows, base = [], 0
            for (_, _, want), (_, _, places) in zip(entries, ordered):
                rows += [base + places.index(p) for p in want]
                base += len(places)
            host = logits.cpu().numpy()[rows].astype("<f4")
            host.tofile(os.path.join(args.out, f"{step['step']}.f32"))
        model.check_health()
        print(f"done {step['step']}", file=out, flush=True)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    add_arguments(ap)
    return run(ap.parse_args(argv))
