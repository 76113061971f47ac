"""Decode and prefill throughput of a looped dense-weight decoder (Pesedra) beside the plain affine-u4 decoder
at equal sizes, and both designs' kernels against their rooflines.

Random weights.  Sizes are width / feed-forward / query x key heads x head size; the looped decoder has five
layers of which three run twice (eight layer runs), the plain one eight layers.  Kernels are timed as
``kernel_bench`` times everything: a recorded pass over operand sets larger than L2, replayed between events.
"""
from __future__ import annotations

import ctypes as C
import json
import os
import time

import numpy as np

from . import capi, checkpoint, kernel_bench, package, pesedra

SIZES = {"2048": (2048, 6144, 16, 4, 128), "4096": (4096, 12288, 32, 8, 128), "5120": (5120, 17408, 40, 8, 128)}
WINDOW, POOL, VOCAB, CHUNK = 1024, 16, 32768, 512


def peak_tflops() -> float:
    path = os.path.join(kernel_bench.ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            return float(json.load(f)["bf16_tflops"])
    return 1590.0


def random_model(width, ff, n_q, n_kv, d, positions):
    """Configuration and tensors of a looped decoder; one random tensor per shape, shared by the layers' names."""
    layer = {"type": "attention", "mixer": {"heads": n_q, "kv_heads": n_kv, "dim": d, "vdim": d, "scale": d ** -0.5, "softcap": 20.0, "mask": {"size": WINDOW, "pool": POOL}},
             "mlp": {"kind": "dense", "ff": ff}}
    config = pesedra.parse({"architecture": "Pesedra", "embedding": {"scale": 1.0}, "layers": [layer] * 5, "loop": {"start": 1, "stop": 4, "times": 2}, "max_positions": positions,
                            "norm": {"eps": 1e-6}, "vocab": VOCAB, "width": width})
    rng, made, out = np.random.default_rng(1), {}, {}
    for name, shape in pesedra.tensor_shapes(config).items():
        if shape not in made:
            bits = rng.integers(0, 1 << 16, shape, dtype=np.uint16)
            exponent = 127 - int(np.ceil(np.log2(max(shape[-1], 2)) / 2)) if len(shape) == 2 else 127
            made[shape] = np.asarray((bits & np.uint16(0x807F if len(shape) == 2 else 0x007F)) | np.uint16(exponent << 7))
        out[name] = ("BF16", made[shape])
    return config, checkpoint.TensorFile(out)


def time_decoder(ctx, dec, prompt, steps, warmup, prefill):
    """Prefill (wall clock around the synchronous call, best of three) and decode (device events around graph replays)."""
    best = None
    for _ in range(3):
        ctx.synchronize()
        t0 = time.perf_counter()
        prefill(prompt)
        ctx.synchronize()
        dt = time.perf_counter() - t0
        best = dt if best is None else min(best, dt)
    dec.build_graph()
    dec.graph_seed([int(prompt[-1])], len(prompt))
    dec.graph_decode(warmup, read=False)
    ctx.synchronize()
    ms = C.c_float(0)
    ctx.call("timer_start")
    dec.graph_decode(steps, read=False)
    ctx._check(ctx.lib.smelt_cuda_timer_stop(ctx.h, C.byref(ms)))
    return {"prefill_ms": round(best * 1e3, 3), "prefill_tok_s": round(len(prompt) / best, 1), "decode_ms_per_token": round(ms.value / steps, 4),
            "decode_tok_s": round(steps * 1e3 / ms.value, 1), "launches_per_token": int(ctx.lib.smelt_cuda_last_launch_count(ctx.h))}


def models(size, steps, warmup, prompt_len):
    width, ff, n_q, n_kv, d = SIZES[size]
    positions = prompt_len + warmup + steps + 16
    prompt = np.random.default_rng(3).integers(0, VOCAB, prompt_len).astype(np.int32)
    out = {}
    ctx = capi.Context(0)
    config, tensors = random_model(width, ff, n_q, n_kv, d, positions)
    dec = pesedra.decoder(ctx, config, tensors, max_chunk=CHUNK)
    per_run = (n_q + 2 * n_kv) * d * width + 2 * ff * width + n_q * d * width
    keys = WINDOW + (prompt_len - WINDOW) // POOL
    token_bytes = 2 * (8 * per_run + 2 * 2 * width * width + VOCAB * width) + 8 * 2 * n_kv * d * 2 * keys
    r = time_decoder(ctx, dec, prompt, steps, warmup, dec.prefill)
    r["bytes_per_token"], r["decode_gbs"] = token_bytes, round(token_bytes / (r["decode_ms_per_token"] * 1e6), 1)
    out["pesedra"] = r
    ctx.close()
    ctx = capi.Context(0)
    cfg = package.DecoderConfig(layers=8, hidden=width, inter=ff, n_q=n_q, n_kv=n_kv, head_dim=d, vocab=VOCAB)
    image, desc, layers = package.build_image(package.SyntheticPackage(cfg, 0))
    dec = package.Decoder(ctx, image, desc, layers, positions, fuse_residual=3)
    per_layer = (2 * n_q + 2 * n_kv) * d * width + 3 * ff * width
    token_bytes = 8 * per_layer * 0.5625 + 2 * VOCAB * width + 8 * 2 * n_kv * d * 2 * prompt_len
    r = time_decoder(ctx, dec, prompt, steps, warmup, lambda p: dec.prefill(p, 0, CHUNK))
    r["bytes_per_token"], r["decode_gbs"] = token_bytes, round(token_bytes / (r["decode_ms_per_token"] * 1e6), 1)
    out["plain_u4"] = r
    ctx.close()
    return out


def kernels(size, reps=10):
    """Each kernel of the looped decoder beside the plain decoder's like kernel: share of the roofline (the larger of
    bytes over the measured copy bandwidth and operations over the measured bf16 rate, over the time)."""
    width, ff, n_q, n_kv, d = SIZES[size]
    b, flops_peak = kernel_bench.Bench(reps, quiet=True), peak_tflops()
    qkv, position = (n_q + 2 * n_kv) * d, 3 * WINDOW - 3
    keys = WINDOW + (position + 1 - WINDOW) // POOL

    def share(pick):
        b.rows.clear()
        pick()
        r = b.rows[-1]
        bound = max(r["bytes_per_launch"] / (b.peak * 1e9), r.get("tflops", 0.0) * r["us_per_launch"] * 1e-6 / flops_peak)
        return {"kernel": r["kernel"], "shape": r["shape"], "us": r["us_per_launch"], "gbs": r["achieved_gbs"], **({"tflops": r["tflops"]} if "tflops" in r else {}),
                "of_roofline": round(bound / (r["us_per_launch"] * 1e-6), 4)}

    pairs = {
        "decode, input projection": (lambda: b.dense_matvec(size, qkv + ff, width, split=qkv), lambda: b.affine(size, ff, width, 1, "gate_up")),
        "decode, output projection": (lambda: b.dense_matvec(size, width, n_q * d + ff, add=True), lambda: b.affine(size, width, ff, 1, "add")),
        "decode, loop entry": (lambda: b.dense_matvec(size, width, 2 * width), lambda: b.affine(size, width, width, 1, "matvec")),
        "decode, head": (lambda: b.dense_matvec(size, VOCAB, width), lambda: b.lm_head(size, VOCAB, width)),
        "decode, attention": (lambda: b.window(size, n_q, n_kv, d, WINDOW, POOL, position), lambda: b.attention(size, n_q, n_kv, d, keys, 1)),
        f"{CHUNK} positions, input projection": (lambda: b.dense_gemm(size, qkv + ff, width, CHUNK, split=qkv), lambda: b.affine(size, ff, width, CHUNK, "gate_up")),
        f"{CHUNK} positions, output projection": (lambda: b.dense_gemm(size, width, n_q * d + ff, CHUNK, add=True), lambda: b.affine(size, width, ff, CHUNK, "add")),
        f"{CHUNK} positions, attention": (lambda: b.window(size, n_q, n_kv, d, WINDOW, POOL, position, m=CHUNK), lambda: b.attention_prefill(size, n_q, n_kv, d, CHUNK, keys - CHUNK)),
    }
    out = []
    for name, (ours, like) in pairs.items():
        a, c = share(ours), share(like)
        out.append({"step": name, "pesedra": a, "plain_u4": c, "roofline_ratio": round(a["of_roofline"] / c["of_roofline"], 3)})
    b.ctx.close()
    return out


def run(sizes, steps, warmup, prompt_len=2048):
    out = {}
    for size in sizes:
        out[size] = {"size": dict(zip(("width", "ff", "heads", "kv_heads", "dim"), SIZES[size])), "kernels": kernels(size), **models(size, steps, warmup, prompt_len)}
    return out
