"""Decode and prefill throughput of a stack of latent attention, time mixing and expert layers (Kesedra)
beside the looped dense-weight decoder (Pesedra) at equal sizes, and both designs' kernels against their rooflines.

    python -m smelt_b200.stack_bench --size 4096 --only "time mixing recurrence" [--alone] [--reps 10]

times the kernels of the steps whose name contains --only (profiler captures); ``bench.py --model kesedra`` runs all.

Random weights.  Sizes are width / feed-forward / heads; eight layers of each design (Kesedra: latent attention +
dense, latent attention on the same cache + experts, time mixing + dense, time mixing + experts, twice).  Kernels are
timed as ``kernel_bench`` times everything: a recorded pass over operand sets larger than L2, replayed between events.
"""
from __future__ import annotations

import argparse
import ctypes as C
import json

import numpy as np

from . import capi, checkpoint, dense_bench, kernel_bench, kesedra, pesedra
from .dense_bench import CHUNK, VOCAB, WINDOW

# width -> feed-forward, attention heads, query latent, inner size of the decay, expert feed-forward
SIZES = {"2048": (6144, 16, 768, 64, 768), "4096": (12288, 32, 1536, 64, 1536), "5120": (17408, 40, 1536, 96, 2176)}
DIM, ROT, RANK, WKV_DIM, EXPERTS, TOP = 128, 64, 512, 64, 16, 4


def random_model(size):
    """Configuration and tensors; one random tensor per shape, shared by the layers' names."""
    width = int(size)
    ff, heads, q_rank, rank, expert_ff = SIZES[size]
    latent = {"dim": DIM, "heads": heads, "kv_rank": RANK, "mask": {"size": WINDOW}, "q_rank": q_rank, "rot": {"base": 10000.0, "dims": ROT}, "rot_dim": ROT, "scale": (DIM + ROT) ** -0.5, "vdim": DIM}
    wkv = {"dim": WKV_DIM, "heads": width // WKV_DIM}
    dense, moe = {"kind": "dense", "ff": ff}, {"kind": "moe", "expert": {"ff": expert_ff, "limit": 7.0}, "router": {"experts": EXPERTS, "top": TOP}}
    layers = []
    for at in (0, 4):
        layers += [{"type": "latent_attention", "mixer": latent, "mlp": dense}, {"type": "latent_attention", "mixer": {**latent, "kv_from": at}, "mlp": moe},
                   {"type": "wkv", "mixer": wkv, "mlp": dense}, {"type": "wkv", "mixer": wkv, "mlp": moe}]
    config = kesedra.parse({"architecture": "Kesedra", "embedding": {"scale": 1.0}, "layers": layers, "norm": {"eps": 1e-6}, "vocab": VOCAB, "width": width})
    rng, made, out = np.random.default_rng(1), {}, {}
    for name, shape in kesedra.tensor_shapes(config, lambda i: rank).items():
        if shape not in made:
            bits = rng.integers(0, 1 << 16, shape, dtype=np.uint16)
            exponent = 127 - int(np.ceil(np.log2(max(shape[-1], 2)) / 2)) if len(shape) == 2 else 120
            made[shape] = np.asarray((bits & np.uint16(0x807F)) | np.uint16(exponent << 7))
        out[name] = ("BF16", made[shape])
    return config, checkpoint.TensorFile(out)


def token_bytes(size, position):
    """Weights, cache and state that a decoded token reads (and the state it writes)."""
    width = int(size)
    ff, heads, q_rank, rank, expert_ff = SIZES[size]
    keys = min(WINDOW, position + 1)
    latent = (q_rank * width + heads * (DIM + ROT) * q_rank + 2 * heads * DIM * RANK + width * heads * DIM) * 2 + keys * (RANK + ROT) * 2
    wkv = (5 * width * width + 2 * rank * width) * 2 + 2 * width * WKV_DIM * 4
    dense, experts = 2 * ff * width * 2, (EXPERTS * width + 3 * TOP * expert_ff * width) * 2
    return 2 * (2 * latent + (RANK + ROT) * width * 2 + 2 * wkv + 2 * dense + 2 * experts) + VOCAB * width * 2


def models(size, steps, warmup, prompt_len):
    positions = prompt_len + warmup + steps + 16
    prompt = np.random.default_rng(3).integers(0, VOCAB, prompt_len).astype(np.int32)
    out = {}
    ctx = capi.Context(0)
    config, tensors = random_model(size)
    dec = kesedra.decoder(ctx, config, tensors, max_chunk=CHUNK)
    r = dense_bench.time_decoder(ctx, dec, prompt, steps, warmup, dec.prefill)
    r["bytes_per_token"] = token_bytes(size, prompt_len)
    r["decode_gbs"] = round(r["bytes_per_token"] / (r["decode_ms_per_token"] * 1e6), 1)
    out["kesedra"] = r
    ctx.close()
    ctx = capi.Context(0)
    width, ff, n_q, n_kv, d = dense_bench.SIZES[size]
    config, tensors = dense_bench.random_model(width, ff, n_q, n_kv, d, positions)
    dec = pesedra.decoder(ctx, config, tensors, max_chunk=CHUNK)
    out["pesedra"] = dense_bench.time_decoder(ctx, dec, prompt, steps, warmup, dec.prefill)
    ctx.close()
    return out


class Bench(kernel_bench.Bench):
    """The cases of this design's kernels."""

    def weights(self, tag, rows, cols, n):
        return [self.ctx.to_device(self.bf16_weights(tag, rows, cols)) for _ in range(n)]

    def matvec(self, config, kind, rows, cols, groups=0, bias=False):
        ctx, n = self.ctx, kernel_bench.copies_for(rows * cols * 2)
        w = self.weights(f"sm{rows}", rows, cols, n)
        f = lambda k, v=1.0: ctx.to_device(np.full(k, v, np.float32))
        b = lambda k: ctx.to_device(np.full(k, 0x3D00, np.uint16))
        bufs = {"x": f(cols), "y": f(cols), "post_norm": b(cols), "norm": b(cols), "before": f(cols), "mu": b(5 * cols), "bias": b(rows), "x_out": f(cols), "h_out": f(cols), "out": f(rows)}
        a = capi.StackMatvecArgs(input=kind, rows=rows, cols=cols, width=cols, group_rows=groups, act=1 if bias else 0, eps=1e-6, **{k: v.ptr for k, v in bufs.items()})
        if kind in (capi.MATVEC_PLAIN, capi.MATVEC_NORM):
            a.y = None
        if not bias:
            a.bias = None

        def enqueue():
            for wi in w:
                a.w = wi.ptr
                ctx.call("stack_matvec", C.byref(a), 5)
        alg = rows * cols * 2 + rows * 4 + cols * 4 * (3 if kind >= capi.MATVEC_RESIDUAL else 1)
        self.run(config, "stack_matvec (" + ("plain", "norm", "residual, norms", "residual, norms, shift")[kind] + ")", f"{rows}x{cols}", 1, alg, n, enqueue)
        for x in (*w, *bufs.values()):
            x.free()

    def experts_matvec(self, config, out, width, ff):
        """The chosen experts' product of a decode step."""
        ctx = self.ctx
        rows, cols = (width, ff) if out else (2 * ff, width)
        n = kernel_bench.copies_for(TOP * rows * cols * 2, cap=12)
        w = self.weights(f"ex{rows}", EXPERTS * rows, cols, n)
        x, y = ctx.to_device(np.ones(TOP * cols, np.float32)), ctx.alloc(TOP * rows * 4)
        logits, chosen = ctx.to_device(np.arange(EXPERTS, dtype=np.float32)[::-1].copy()), ctx.to_device(np.array([[3 * k, 0x3E800000] for k in range(TOP)], np.int32))
        a = capi.StackMatvecArgs(input=capi.MATVEC_EXPERTS_OUT if out else capi.MATVEC_EXPERTS_IN, rows=rows, cols=cols, experts=EXPERTS, top=TOP, limit=7.0, x=x.ptr, out=y.ptr, logits=logits.ptr,
                                 chosen=chosen.ptr)

        def enqueue():
            for wi in w:
                a.w = wi.ptr
                ctx.call("stack_matvec", C.byref(a), 5)
        self.run(config, "stack_matvec (experts, " + ("down)" if out else "choice, gate and up)"), f"{TOP} of {EXPERTS} x {rows}x{cols}", 1, TOP * rows * cols * 2, n, enqueue)
        for b in (*w, x, y, logits, chosen):
            b.free()

    def latent(self, config, heads, position, m=1, part=None):
        """A decode step's attention (query, scores, values; one of them with `part`) or a prompt chunk's tiled attention."""
        ctx, pos0 = self.ctx, position + 1 - m
        ring = -(-(WINDOW + m) // 64) * 64
        cache = ring * (RANK + ROT) * 2 if m == 1 else ring * (heads * 2 * DIM + ROT) * 2
        keys = min(position + 1, WINDOW + m - 1)
        proj = heads * 2 * DIM * RANK * 2
        if m == 1:
            alg = {None: proj + keys * (RANK + ROT) * 2, "query": proj / 2, "scores": keys * (RANK + ROT) * 2, "values": proj / 2}[part]
        else:
            alg = keys * (heads * 2 * DIM + ROT) * 2 + m * heads * (2 * DIM + ROT) * 2
        n = kernel_bench.copies_for(cache + (proj if m == 1 else 0), cap=48)
        sets = []
        for _ in range(n):
            if m == 1:
                sets.append((ctx.to_device(self.bf16_weights("lc", ring, RANK)), ctx.to_device(self.bf16_weights("lr", ring, ROT)), ctx.to_device(self.bf16_weights("lp", heads * 2 * DIM, RANK))))
            else:
                sets.append((ctx.to_device(self.bf16_weights("lk", ring, heads * 2 * DIM)), ctx.to_device(self.bf16_weights("lr", ring, ROT)), None))
        f = lambda k: ctx.to_device(np.ones(k, np.float32))
        shared = {"u": f(64 + RANK + ROT), "kv_norm": ctx.to_device(np.full(RANK, 0x3F80, np.uint16)), "rot_freq": ctx.to_device(10000.0 ** (-np.arange(ROT // 2) / (ROT // 2))),
                  "q": f(heads * (DIM + ROT)) if m == 1 else ctx.to_device(self.bf16_weights("lq", m * heads, DIM + ROT)), "qa": f(heads * (RANK + ROT)), "sums": f(64 * heads * RANK),
                  "maxima": f(2 * 64 * heads), "z": f(m * heads * DIM)}
        a = capi.LatentArgs(heads=heads, dim=DIM, rot_dim=ROT, rot_dims=ROT, vdim=DIM, kv_rank=RANK, q_rank=64, own=1, window=WINDOW, ring=ring, scale=0.07, eps=1e-6, m=m, ldu=64 + RANK + ROT,
                            ldz=heads * DIM, decode=int(m == 1), **{k: v.ptr for k, v in shared.items()})

        def enqueue():
            for c, r, p in sets:
                a.rot_ring = r.ptr
                if m > 1:
                    a.kv_rows = c.ptr
                    ctx.call("latent_prefill", C.byref(a), pos0)
                    continue
                a.latent_ring, a.kv_proj = c.ptr, p.ptr
                for step in ("query", "scores", "values"):
                    if part in (None, step):
                        ctx.call("latent_" + step, 0, C.byref(a), position)
        seen = sum(min(i + 1, WINDOW) for i in range(pos0, position + 1))
        flops = 2.0 * heads * (2 * DIM + ROT) * seen if m > 1 else 2.0 * heads * (2 * RANK + ROT) * keys
        self.run(config, f"latent_{part or 'query + scores + values'}" if m == 1 else "latent_prefill", f"{heads} heads x ({DIM} + {ROT}), rank {RANK}, window {WINDOW}, "
                 + (f"position {position}" if m == 1 else f"{m} positions from {pos0}"), 1, alg, n, enqueue, flops=flops)
        for b in (*[x for s in sets for x in s if x], *shared.values()):
            b.free()

    def wkv(self, config, width, rank, m=1):
        ctx, D = self.ctx, WKV_DIM
        heads, rp = width // D, -(-rank // 64) * 64
        state_bytes = heads * D * D * 4
        n = kernel_bench.copies_for(state_bytes + (width * rp * 2 if m == 1 else m * width * 20), cap=64)
        ldu = 4 * width + (rp if m == 1 else 0)
        rng = np.random.default_rng(0)
        u = ctx.to_device(rng.standard_normal(m * ldu).astype(np.float32) * 0.1)
        b = lambda k: ctx.to_device(np.full(k, 0x3D00, np.uint16))
        sets = [(ctx.alloc(state_bytes).fill(0), ctx.to_device(self.bf16_weights("w2", width, rp)), ctx.to_device(np.full(m * width, 0.9, np.float32)) if m > 1 else None) for _ in range(n)]
        shared = {"u": u, "w0": b(width), "bonus": b(width), "norm": b(width), "h": ctx.to_device(np.ones(m * width, np.float32)), "before": ctx.alloc(width * 4), "out": ctx.alloc(m * width * 4)}
        a = capi.WkvArgs(heads=heads, dim=D, rank=rp, ld=width, m=m, ldu=ldu, ldz=width, eps=1e-6, **{k: v.ptr for k, v in shared.items()})

        def enqueue():
            for st, w2, dec in sets:
                a.state, a.w2 = st.ptr, w2.ptr
                if m > 1:
                    a.decay = dec.ptr
                    ctx.call("wkv_prefill", C.byref(a), 1024)
                else:
                    ctx.call("wkv_decode", C.byref(a), 1024)
        alg = 2 * state_bytes + (width * rp * 2 + 5 * width * 4 if m == 1 else m * width * 20)
        self.run(config, "wkv_decode" if m == 1 else "wkv_prefill", f"{heads} heads x {D}, {m} positions", 1, alg, n, enqueue)
        for x in (*[y for s in sets for y in s if y], *shared.values()):
            x.free()

    def gemm(self, config, rows, cols, m, mode=2, groups=0):
        """A chunk's product; groups: rows of each group with activations of its own."""
        ctx = self.ctx
        ng = -(-rows // groups) if groups else 1
        alg = rows * cols * 2 + ng * m * cols * 2 + m * rows * (2 if mode == 2 else 4)
        n = kernel_bench.copies_for(alg, cap=16)
        w = self.weights(f"sg{rows}", rows, cols, n)
        x, y, y1 = ctx.to_device(self.bf16_weights("sgx", ng * m, cols)), ctx.alloc(m * rows * 4).fill(0), ctx.alloc(m * rows * 4).fill(0)
        split = rows // groups * groups if groups else 0 if mode == 2 else rows
        act = 2 if groups else 1 if mode == 2 else 0

        def enqueue():
            for wi in w:
                ctx.call("dense_gemm_ex", 0, mode, wi, x, None, y, y1, rows, cols, m, split, rows, rows, act, groups)
        self.run(config, "dense_gemm " + ("(five inputs, tanh)" if groups else "(squared ReLU)" if mode == 2 else "(fp32)"), f"{rows}x{cols}", m, alg, n, enqueue, flops=2.0 * rows * cols * m)
        for b in (*w, x, y, y1):
            b.free()

    def moe(self, config, width, ff, m, stage):
        ctx = self.ctx
        rng = np.random.default_rng(2)
        n = 2
        up, down = self.weights("mu", EXPERTS * 2 * ff, width, n), self.weights("md", EXPERTS * width, ff, n)
        logits = ctx.to_device(rng.standard_normal((m, EXPERTS)).astype(np.float32))
        pairs = m * TOP
        shared = {"logits": logits, "h": ctx.to_device(self.bf16_weights("mh", m, width)), "chosen": ctx.alloc(pairs * 8), "place": ctx.alloc(pairs * 4), "table": ctx.alloc((1 + EXPERTS + pairs) * 16),
                  "permuted": ctx.alloc(pairs * width * 2), "inner": ctx.alloc(pairs * ff * 2), "rows": ctx.alloc(pairs * width * 4), "y": ctx.alloc(m * width * 4)}
        a = capi.MoeArgs(m=m, experts=EXPERTS, top=TOP, ff=ff, width=width, limit=7.0, up=up[0].ptr, down=down[0].ptr, **{k: v.ptr for k, v in shared.items()})
        ctx.call("moe_rows", 0, C.byref(a), 5, 0)

        def enqueue():
            for i in range(n):
                a.up, a.down = up[i].ptr, down[i].ptr
                ctx.call("moe_rows", 0, C.byref(a), stage, 1)
        alg = {1: m * EXPERTS * 4, 2: m * width * 2 + pairs * width * 2, 3: EXPERTS * 2 * ff * width * 2 + pairs * (width + ff) * 2, 4: EXPERTS * width * ff * 2 + pairs * (ff * 2 + width * 4),
               5: pairs * width * 4 + m * width * 4}[stage]
        flops = {3: 4.0 * pairs * ff * width, 4: 2.0 * pairs * ff * width}.get(stage, 0.0)
        self.run(config, "experts: " + ("choice and permutation", "gather", "gate and up", "down", "weighted sum")[stage - 1], f"{m} x {TOP} of {EXPERTS}, {width} / {ff}", m, alg, n, enqueue, flops=flops)
        for b in (*up, *down, *shared.values()):
            b.free()

    def rows_kernel(self, config, what, width, m):
        """Row kernels of a prompt chunk, over enough chunks to leave L2."""
        ctx = self.ctx
        D, heads = WKV_DIM, width // WKV_DIM
        alg = {"residual_norm": m * width * (4 * 3 + 2), "scalar_norm": m * width * 6, "shift": m * width * (4 + 10), "gate": m * width * (4 + 4 + 2)}[what]
        n = kernel_bench.copies_for(alg, cap=24)
        xs = [ctx.alloc(m * width * 4 * (4 if what == "gate" else 1)).fill(0) for _ in range(n)]
        ys = [ctx.alloc(m * width * 4).fill(0) for _ in range(n)]
        outs = [ctx.alloc(m * width * 2 * (5 if what == "shift" else 1)) for _ in range(n)]
        norm = ctx.to_device(np.full(5 * width, 0x3D00, np.uint16))
        before = ctx.alloc(width * 4).fill(0)

        def enqueue():
            for x, y, o in zip(xs, ys, outs):
                if what == "residual_norm":
                    ctx.call("residual_norm_rows", 0, x, y, norm, norm, None, o, None, width, width, m, 1e-6)
                elif what == "scalar_norm":
                    ctx.call("scalar_norm_rows", 0, x, None, o, width, width, m, 1.0, 1e-6)
                else:
                    a = capi.WkvArgs(heads=heads, dim=D, rank=64, ld=width, m=m, ldu=4 * width, ldz=width, eps=1e-6, u=x.ptr, o=y.ptr, norm=norm.ptr, mu=norm.ptr, before=before.ptr, h=x.ptr, out=o.ptr)
                    if what == "shift":
                        ctx.call("wkv_shift", 0, C.byref(a), 7)
                    else:
                        ctx.call("wkv_gate", 0, C.byref(a))
        self.run(config, what + " rows", f"{m} x {width}", m, alg, n, enqueue)
        for b in (*xs, *ys, *outs, norm, before):
            b.free()


def kernels(size, reps=10, only="", alone=False):
    """Each kernel beside Pesedra's (or the DeltaNet mixer's) like kernel: share of the roofline (the larger of bytes over
    the measured copy bandwidth and operations over the measured bf16 rate, over the time).  only: the steps whose name
    contains it; alone: without the like kernels."""
    width = int(size)
    ff, heads, q_rank, rank, expert_ff = SIZES[size]
    b, peak = Bench(reps, quiet=True), dense_bench.peak_tflops()
    n_kv = dense_bench.SIZES[size][3]
    position, in_rows, q_rows, group = 3 * WINDOW - 3, q_rank + RANK + ROT, heads * (DIM + ROT), width
    rp = -(-rank // 64) * 64

    def share(pick):
        b.rows.clear()
        pick()
        r = b.rows[-1]
        bound = max(r["bytes_per_launch"] / (b.peak * 1e9), r.get("tflops", 0.0) * r["us_per_launch"] * 1e-6 / peak)
        return {"kernel": r["kernel"], "shape": r["shape"], "us": r["us_per_launch"], "gbs": r["achieved_gbs"], **({"tflops": r["tflops"]} if "tflops" in r else {}),
                "of_roofline": round(bound / (r["us_per_launch"] * 1e-6), 4)}

    mv = lambda kind, rows, cols, **kw: (lambda: b.matvec(size, kind, rows, cols, **kw), lambda: b.dense_matvec(size, rows, cols))
    gm = lambda rows, cols, mode=0, **kw: (lambda: b.gemm(size, rows, cols, CHUNK, mode, **kw), lambda: b.dense_gemm(size, rows, cols, CHUNK, split=rows))
    pairs = {
        "decode, latent input projection": mv(capi.MATVEC_RESIDUAL, in_rows, width),
        "decode, query projection": mv(capi.MATVEC_NORM, q_rows, q_rank),
        "decode, latent attention": (lambda: b.latent(size, heads, position), lambda: b.window(size, heads, n_kv, DIM, WINDOW, dense_bench.POOL, position)),
        "decode, attention output projection": mv(capi.MATVEC_PLAIN, width, heads * DIM),
        "decode, time mixing projection": mv(capi.MATVEC_SHIFT, 4 * group + rp, width, groups=group),
        "decode, time mixing step": (lambda: b.wkv(size, width, rank), lambda: b.deltanet(size, 128, 32, 16, 1)),
        "decode, feed-forward up": mv(capi.MATVEC_RESIDUAL, ff, width, bias=True),
        "decode, feed-forward down": mv(capi.MATVEC_PLAIN, width, ff),
        "decode, router": mv(capi.MATVEC_RESIDUAL, EXPERTS, width),
        "decode, experts gate and up": (lambda: b.experts_matvec(size, False, width, expert_ff), lambda: b.dense_matvec(size, 2 * TOP * expert_ff, width)),
        "decode, experts down": (lambda: b.experts_matvec(size, True, width, expert_ff), lambda: b.dense_matvec(size, width, TOP * expert_ff)),
        "decode, head": mv(capi.MATVEC_RESIDUAL, VOCAB, width),
        f"{CHUNK} positions, latent input projection": gm(in_rows, width),
        f"{CHUNK} positions, query projection": gm(q_rows, q_rank, 2),
        f"{WINDOW + CHUNK} rows, keys and values of the ring": (lambda: b.gemm(size, 2 * heads * DIM, RANK, WINDOW + CHUNK, 2), lambda: b.dense_gemm(size, 2 * heads * DIM, RANK, WINDOW + CHUNK)),
        f"{CHUNK} positions, latent attention": (lambda: b.latent(size, heads, position, m=CHUNK), lambda: b.window(size, heads, n_kv, DIM, WINDOW, dense_bench.POOL, position, m=CHUNK)),
        f"{CHUNK} positions, attention output projection": gm(width, heads * DIM),
        f"{CHUNK} positions, time mixing projections": gm(4 * group + rp, width, 3, groups=group),
        f"{CHUNK} positions, time mixing recurrence": (lambda: b.wkv(size, width, rank, m=CHUNK), lambda: b.deltanet(size, 128, 32, 16, CHUNK)),
        f"{CHUNK} positions, feed-forward up": gm(ff, width, 2),
        f"{CHUNK} positions, feed-forward down": gm(width, ff),
        f"{CHUNK} positions, experts gate and up": (lambda: b.moe(size, width, expert_ff, CHUNK, 3), lambda: b.dense_gemm(size, 2 * expert_ff * TOP, width, CHUNK)),
        f"{CHUNK} positions, experts down": (lambda: b.moe(size, width, expert_ff, CHUNK, 4), lambda: b.dense_gemm(size, width, expert_ff * TOP, CHUNK)),
        f"{CHUNK} positions, experts choice and permutation": (lambda: b.moe(size, width, expert_ff, CHUNK, 1), None),
        f"{CHUNK} positions, experts gather": (lambda: b.moe(size, width, expert_ff, CHUNK, 2), lambda: b.rows_kernel(size, "scalar_norm", width, CHUNK)),
        f"{CHUNK} positions, experts weighted sum": (lambda: b.moe(size, width, expert_ff, CHUNK, 5), lambda: b.rows_kernel(size, "scalar_norm", width, CHUNK)),
        f"{CHUNK} positions, residual and norms": (lambda: b.rows_kernel(size, "residual_norm", width, CHUNK), lambda: b.rows_kernel(size, "scalar_norm", width, CHUNK)),
        f"{CHUNK} positions, token shift and mixes": (lambda: b.rows_kernel(size, "shift", width, CHUNK), lambda: b.rows_kernel(size, "scalar_norm", width, CHUNK)),
        f"{CHUNK} positions, head norm and gate": (lambda: b.rows_kernel(size, "gate", width, CHUNK), lambda: b.rows_kernel(size, "scalar_norm", width, CHUNK)),
    }
    out = []
    for name, (ours, like) in pairs.items():
        if only and only not in name:
            continue
        a = share(ours)
        if like is None or alone:
            out.append({"step": name, "kesedra": a})
            continue
        c = share(like)
        out.append({"step": name, "kesedra": a, "like": c, "roofline_ratio": round(a["of_roofline"] / c["of_roofline"], 3)})
    b.ctx.close()
    return out


def run(sizes, steps, warmup, prompt_len=2048):
    return {size: {"size": {"width": int(size), **dict(zip(("ff", "heads", "q_rank", "decay_rank", "expert_ff"), SIZES[size]))}, "kernels": kernels(size),
                   **models(size, steps, warmup, prompt_len)} for size in sizes}


def main():
    ap = argparse.ArgumentParser(prog="smelt_b200.stack_bench")
    ap.add_argument("--size", default="4096", choices=list(SIZES))
    ap.add_argument("--only", default="")
    ap.add_argument("--reps", type=int, default=10)
    ap.add_argument("--alone", action="store_true", help="without the like kernels")
    args = ap.parse_args()
    for row in kernels(args.size, args.reps, args.only, args.alone):
        print(json.dumps(row), flush=True)


if __name__ == "__main__":
    main()
