"""Greedy generation from a model folder.

    python -m smelt_b200.generate --model DIR --prompt 12,7,301 --tokens 32 [--dtype bfloat16|float32]

--prompt takes token ids separated by commas, or @FILE with ids separated by white space or commas.
Prints the generated ids on one line.
"""
from __future__ import annotations

import argparse
import re
import sys


def parse_ids(text: str) -> list[int]:
    if text.startswith("@"):
        with open(text[1:]) as f:
            text = f.read()
    return [int(t) for t in re.split(r"[,\s]+", text) if t]


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="smelt_b200.generate", description="Greedy generation from a model folder.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", required=True, help="token ids: 1,2,3 or @FILE")
    ap.add_argument("--tokens", type=int, default=32, help="ids to generate")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="activations and caches")
    ap.add_argument("--max-chunk", type=int, default=512, help="positions per prompt chunk")
    args = ap.parse_args(argv)
    prompt = parse_ids(args.prompt)
    if not prompt or args.tokens < 0:
        ap.error("the prompt needs at least one id, and --tokens cannot be negative")
    from . import capi, checkpoint

    decoder = checkpoint.open_model(capi.Context(0), args.model, precision=args.dtype, max_chunk=args.max_chunk)
    print(" ".join(str(int(t)) for t in decoder.generate(prompt, args.tokens)[:, 0]), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
