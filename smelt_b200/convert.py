"""Writes a model folder (config.json and model.safetensors) as a ``.smeltpkg`` directory.

    python -m smelt_b200.convert --model DIR --out X.smeltpkg [--dtype bfloat16|float32] [--capacity N] [--max-chunk N]
"""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="smelt_b200.convert", description="Write a model folder as a .smeltpkg directory.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--out", required=True, help="the package directory to write")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="activations and caches")
    ap.add_argument("--capacity", type=int, default=0, help="positions (0: all the model has)")
    ap.add_argument("--max-chunk", type=int, default=512, help="positions per prompt chunk")
    args = ap.parse_args(argv)
    from . import checkpoint

    checkpoint.convert(args.model, args.out, precision=args.dtype, capacity=args.capacity, max_chunk=args.max_chunk)
    return 0


if __name__ == "__main__":
    sys.exit(main())
