"""Replays a trace of token steps through a model folder and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one JSON line: {"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}.
Its tokens follow what earlier steps fed for the same id; "want" lists places among them whose logits go
to DIR/<step>.f32 (fp32, little-endian, [wanted, vocab]); "end" lists the ids that are finished.  "done <step>"
is printed after each.  One sequence lives at a time, as in the decoder that runs it.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


class Replay:
    """Feeds steps to one decoder; keeps the live id and how many tokens it has."""

    def __init__(self, decoder):
        self.decoder, self.live, self.length = decoder, None, 0

    def step(self, entries, end) -> np.ndarray:
        rows = []
        for e in entries:
            if self.live is None:
                self.live, self.length = e["id"], 0
            elif self.live != e["id"]:
                raise ValueError(f"request {e['id']!r} while {self.live!r} is live: this decoder holds one sequence")
            rows.append(self.decoder.feed(e["tokens"], self.length, e.get("want", ())))
            self.length += len(e["tokens"])
        for name in end:
            if name == self.live:
                self.live, self.length = None, 0
        return np.concatenate(rows) if rows else np.zeros((0, 0), np.float32)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="activations and caches")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens a live request holds (window caches do not grow with it: not needed)")
    ap.add_argument("--max-chunk", type=int, default=512, help="positions per prompt chunk")
    args = ap.parse_args(argv)
    from . import capi, checkpoint

    replay = Replay(checkpoint.open_model(capi.Context(0), args.model, precision=args.dtype, max_chunk=args.max_chunk))
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step.get("entries", []), step.get("end", []))
        if logits.shape[0]:
            logits.astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    if replay.decoder.ctx.device_error_flags():
        raise RuntimeError("a kernel's bounded wait gave up")
    return 0
