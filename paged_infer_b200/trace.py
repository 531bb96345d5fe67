"""Replay of a recorded schedule: given token ids go through the engine's batched step, step by step, and the logits that
are asked for are written out.  See ``bin/trace_run``."""
from __future__ import annotations

import argparse
import itertools
import json
import os
import sys

import numpy as np

BLOCK = 16
SLOTS = 4            # live requests at any time
ROUND = 64           # a request's tokens are counted in multiples of this


def parse(argv):
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed given token ids through a model and write logits.  Steps are read from standard "
                                 "input, one JSON object a line: {\"step\": n, \"entries\": [{\"id\", \"tokens\", \"want\"}], \"end\": [ids]}.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", required=True, type=int, help="most tokens that live requests hold at any time")
    return ap.parse_args(argv)


def main(argv=None) -> int:
    args = parse(argv)
    from . import api, registry
    from .engine import Engine

    if args.dtype not in registry.FAMILIES[registry.family_of(registry.read_config(args.model))].dtypes:
        print(f"this model family does not compute in {args.dtype}", file=sys.stderr)
        return 3
    ctx = api.Context(0)
    tokens = max(args.max_tokens, ROUND)
    model = registry.load(ctx, args.model, args.dtype, max_rows=tokens)
    engine = Engine(ctx, model, num_blocks=(tokens + BLOCK - 1) // BLOCK, block_size=BLOCK, prefix_cache=False, state_slots=SLOTS)
    numbers, fresh = {}, itertools.count()   # the engine's number of every live request; never given twice
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        for e in step["entries"]:
            if e["id"] not in numbers:
                numbers[e["id"]] = next(fresh)
        entries = [(numbers[e["id"]], e["tokens"], e.get("want", [])) for e in step["entries"]]
        logits = engine.feed(entries)
        if len(logits):
            np.ascontiguousarray(logits, "<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        for i in step.get("end", []):
            if i in numbers:
                engine.end(numbers.pop(i))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
