"""Command line: ``python -m paged_infer_b200 generate --model DIR --tokens 1,2,3 [--tokens ...]`` prints the greedy
continuation of every prompt (token ids, one line each), ``... info --model DIR`` what the checkpoint is."""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="paged_infer_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy continuations of token-id prompts")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    g.add_argument("--tokens", action="append", required=True, help="comma-separated token ids of one prompt; may be given several times")
    g.add_argument("--max-tokens", type=int, default=16)
    g.add_argument("--dtype", choices=["bfloat16", "float32"])
    g.add_argument("--quantization", choices=["f32", "int8"], default="f32", help="Llama: int8 weight-only projections")
    g.add_argument("--max-rows", type=int, default=512, help="tokens one batched step can take")
    g.add_argument("--block-size", type=int, default=16)
    g.add_argument("--eos", type=int)
    i = sub.add_parser("info", help="model family and sizes of a checkpoint folder")
    i.add_argument("--model", required=True)
    args = ap.parse_args(argv)

    from . import registry
    if args.command == "info":
        config = registry.read_config(args.model)
        name = registry.family_of(config)
        print(f"{name}: computes in {', '.join(registry.FAMILIES[name].dtypes)}")
        return 0
    from . import api
    from .engine import Engine
    prompts = [[int(t) for t in p.split(",")] for p in args.tokens]
    ctx = api.Context(0)
    model = registry.load(ctx, args.model, args.dtype, args.max_rows, args.quantization)
    blocks = sum((len(p) + args.max_tokens) // args.block_size + 1 for p in prompts)
    engine = Engine(ctx, model, num_blocks=blocks, block_size=args.block_size, eos=args.eos, state_slots=len(prompts))
    for out in engine.generate(prompts, args.max_tokens):
        print(",".join(str(t) for t in out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
