"""Kesedra on the GPU against the float64 restatement: each kernel alone, then whole models through the
framework's loader, tables, graph and trace replay."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import kesedra_cases as cases
from oracle import kesedra as ref
from smelt_b200 import capi, checkpoint, package
from test_gpu_pesedra import pad_to, put, row_elems, run_cuts, run_cuts_from, seen_as, take, worst, worst_row

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PRECISIONS = ["bfloat16", "float32"]
CODE = package.DenseDecoder.PRECISIONS
EXACT = 3e-5  # of worst(): fp32 sums in another order


@pytest.fixture(scope="module")
def ctx():
    c = capi.Context(0)
    yield c
    assert c.device_error_flags() == 0
    c.close()


def f32(ctx, a):
    return put(ctx, a, "float32")


def padded(a, *shape):
    return np.pad(a, [(0, n - s) for s, n in zip(a.shape, shape)])


# ── matrix-vector products ──────────────────────────────────────────────────
def matvec(ctx, kind, w, x, out_rows, position=3, **kw):
    """Runs ``stack_matvec``; keyword buffers may be arrays (bf16 where a weight) or device buffers."""
    weights = ("post_norm", "norm", "mu", "bias")
    bufs = {k: v if isinstance(v, capi.DeviceBuffer) else put(ctx, v) if k in weights else f32(ctx, v) for k, v in {"w": w, "x": x, **kw}.items() if isinstance(v, (np.ndarray, capi.DeviceBuffer))}
    if isinstance(w, np.ndarray):
        bufs["w"] = put(ctx, w)
    out = f32(ctx, np.full(out_rows + 2, 9.0))
    plain = {k: v for k, v in kw.items() if k not in bufs}
    a = capi.StackMatvecArgs(input=kind, out=out.ptr, **plain, **{k: v.ptr for k, v in bufs.items()})
    ctx.call("stack_matvec", C.byref(a), position)
    got = out.download(np.float32, out_rows + 2)
    assert (got[out_rows:] == 9.0).all()
    return got[:out_rows]


@pytest.mark.parametrize("rows,cols", [(1, 64), (37, 320), (1000, 4096), (4099, 192), (130, 16384)])
def test_matvec_plain_norm_and_bias(ctx, rows, cols):
    g = np.random.default_rng(rows + cols)
    w, x, width = cases.round_bf16(g.standard_normal((rows, cols)) / np.sqrt(cols)), g.standard_normal(cols), cols - 3
    x[width:] = 0
    norm, bias = cases.round_bf16(1 + 0.3 * g.standard_normal(cols)), cases.round_bf16(g.standard_normal(rows))
    assert worst(matvec(ctx, capi.MATVEC_PLAIN, w, x, rows, rows=rows, cols=cols, width=width), ref.linear(w, x)) < EXACT
    want = ref.linear(w, x) + bias
    assert worst(matvec(ctx, capi.MATVEC_PLAIN, w, x, rows, rows=rows, cols=cols, width=width, bias=bias), want) < EXACT
    assert worst(matvec(ctx, capi.MATVEC_PLAIN, w, x, rows, rows=rows, cols=cols, width=width, bias=bias, act=1), np.maximum(want, 0) ** 2) < EXACT
    h = np.zeros(cols)
    h[:width] = ref.plain_norm(x[:width], norm[:width], 1e-3)
    assert worst(matvec(ctx, capi.MATVEC_NORM, w, x, rows, rows=rows, cols=cols, width=width, norm=norm, eps=1e-3), ref.linear(w, h)) < EXACT


def stream_case(g, cols, width):
    x, y = np.zeros(cols), np.zeros(cols)
    x[:width], y[:width] = g.standard_normal(width), 5 * g.standard_normal(width)
    post, norm = np.zeros(cols), np.zeros(cols)
    post[:width], norm[:width] = cases.round_bf16(0.4 * g.standard_normal((2, width)))
    s = x[:width] + ref.zero_centred_norm(y[:width], post[:width], 1e-4)
    return x, y, post, norm, s


@pytest.mark.parametrize("rows,cols,width", [(5, 64, 64), (300, 128, 70), (2000, 4096, 4096), (61, 8192, 8100)])
def test_matvec_on_the_residual_stream(ctx, rows, cols, width):
    g = np.random.default_rng(rows)
    x, y, post, norm, s = stream_case(g, cols, width)
    w = cases.round_bf16(g.standard_normal((rows, cols)) / np.sqrt(cols))
    for with_y in (True, False):
        x_out, h_out = f32(ctx, np.full(cols, 3.0)), f32(ctx, np.full(cols, 3.0))
        kw = {"y": y, "post_norm": post, "x_out": x_out} if with_y else {}
        got = matvec(ctx, capi.MATVEC_RESIDUAL, w, x, rows, rows=rows, cols=cols, width=width, eps=1e-4, norm=norm, h_out=h_out, **kw)
        total = s if with_y else x[:width]
        h = padded(ref.zero_centred_norm(total, norm[:width], 1e-4), cols)
        assert worst(got, ref.linear(w, h)) < EXACT and worst(h_out.download(np.float32, cols), h) < EXACT
        assert worst(x_out.download(np.float32, cols), padded(s, cols) if with_y else np.full(cols, 3.0)) < EXACT


@pytest.mark.parametrize("group,last,cols,width", [(128, 64, 64, 64), (256, 64, 128, 70), (4096, 128, 1024, 1000), (128, 192, 4096, 4096)])
def test_matvec_of_the_shifted_mixes(ctx, group, last, cols, width):
    g = np.random.default_rng(group + cols)
    x, y, post, norm, s = stream_case(g, cols, width)
    rows, before = 4 * group + last, padded(g.standard_normal(width), cols)
    w, mu = cases.round_bf16(g.standard_normal((rows, cols)) / np.sqrt(cols)), padded(cases.round_bf16(g.uniform(0, 1, (5, width))), 5, cols)
    h = ref.zero_centred_norm(s, norm[:width], 1e-4)
    if width < cols:  # the pad columns' weights must not count
        w[:, width:] = 0
    for position in (0, 1, 9):
        h_out, x_out = f32(ctx, np.zeros(cols)), f32(ctx, np.zeros(cols))
        got = matvec(ctx, capi.MATVEC_SHIFT, w, x, rows, position, rows=rows, cols=cols, width=width, eps=1e-4, norm=norm, y=y, post_norm=post, x_out=x_out, h_out=h_out, before=before, mu=mu,
                     group_rows=group)
        shifted = before[:width] if position else np.zeros(width)
        want = np.concatenate([ref.linear(w[n * group:(n + 1) * group if n < 4 else rows, :width], ref.mixed(h, shifted, mu[n, :width])) for n in range(5)])
        assert worst(got, want) < EXACT and worst(h_out.download(np.float32, cols)[:width], h) < EXACT


@pytest.mark.parametrize("experts,top,width,ff", [(1, 1, 64, 64), (5, 2, 128, 64), (40, 7, 320, 128), (64, 64, 64, 64), (16, 4, 2048, 768)])
def test_matvec_of_chosen_experts(ctx, experts, top, width, ff):
    g = np.random.default_rng(experts * 100 + top)
    gate, up = cases.round_bf16(3 * g.standard_normal((2, experts, ff, width)) / np.sqrt(width))
    down, h = cases.round_bf16(g.standard_normal((experts, width, ff)) / np.sqrt(ff)), g.standard_normal(width)
    logits = g.standard_normal(experts).astype(np.float32)
    pairs = np.stack([gate, up], 2).reshape(experts * 2 * ff, width)
    chosen = ctx.alloc(top * 8)
    inner = matvec(ctx, capi.MATVEC_EXPERTS_IN, pairs, h, top * ff, rows=2 * ff, cols=width, experts=experts, top=top, limit=1.25, logits=logits, chosen=chosen)
    picked = chosen.download(np.int32, (top, 2))
    want_e, want_w = ref.route(np.zeros((1, 1)), np.zeros((experts, 1)), logits.astype(np.float64), top)
    assert picked[:, 0].tolist() == want_e[0].tolist() and worst(picked[:, 1].copy().view(np.float32), want_w[0]) < 1e-6
    acts = [ref.expert(h, gate[e], up[e], np.eye(ff), 1.25) * want_w[0, n] for n, e in enumerate(want_e[0])]
    assert worst(inner, np.concatenate(acts)) < EXACT
    got = matvec(ctx, capi.MATVEC_EXPERTS_OUT, down.reshape(-1, ff), inner.astype(np.float32), width, rows=width, cols=ff, experts=experts, top=top, chosen=chosen)
    assert worst(got, sum(ref.linear(down[e], acts[n]) for n, e in enumerate(want_e[0]))) < EXACT


# ── products of a chunk ─────────────────────────────────────────────────────
@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("rows,cols,m", [(5, 64, 2), (130, 192, 33), (700, 1024, 65), (300, 4096, 300), (2048, 128, 17)])
def test_gemm_bias_and_activations(ctx, rows, cols, m, precision):
    g = np.random.default_rng(rows + m)
    w, x, bias = cases.round_bf16(g.standard_normal((rows, cols)) / np.sqrt(cols)), seen_as(g.standard_normal((m, cols)), precision), cases.round_bf16(g.standard_normal(rows))
    z = x @ w.T.astype(np.float64) + bias
    dw, dx, db, split = put(ctx, w), put(ctx, x, precision), put(ctx, bias), rows // 2
    y, y1 = f32(ctx, np.full((m, rows + 1), 7.0)), put(ctx, np.full((m, rows + 2), 7.0), precision)
    call = lambda mode, split, act: ctx.call("dense_gemm_ex", CODE[precision], mode, dw, dx, db, y, y1, rows, cols, m, split, rows + 1, rows + 2, act, 0)
    call(0, rows, 0)
    assert worst(y.download(np.float32, (m, rows + 1))[:, :rows], z) < 1e-4
    call(0, rows, 3)
    assert worst(y.download(np.float32, (m, rows + 1))[:, :rows], np.exp(-np.exp(z))) < 1e-4
    tol = 1e-4 if precision == "float32" else 1 / 256
    for act, f in ((1, lambda v: np.maximum(v, 0) ** 2), (2, np.tanh)):
        for mode, at in ((2, 0), (3, split)):
            call(mode, at, act)
            got = take(y1, (m, rows + 2), precision)
            want = f(z[:, at:])
            assert np.all(np.abs(got[:, :rows - at] - want) <= tol * (np.abs(want) + 0.1)) and (got[:, rows:] == 7.0).all(), (act, mode)
            if at:
                assert worst(y.download(np.float32, (m, rows + 1))[:, :at], z[:, :at]) < 1e-4
    for b in (dw, dx, db, y, y1):
        b.free()


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("group,last,cols,m", [(128, 64, 64, 3), (384, 64, 320, 70), (128, 320, 1024, 300)])
def test_gemm_with_a_group_per_input(ctx, group, last, cols, m, precision):
    g = np.random.default_rng(group + m)
    rows = 4 * group + last
    w, x = cases.round_bf16(g.standard_normal((rows, cols)) / np.sqrt(cols)), seen_as(g.standard_normal((5, m, cols)), precision)
    y, y1 = f32(ctx, np.zeros((m, 4 * group))), put(ctx, np.zeros((m, last)), precision)
    ctx.call("dense_gemm_ex", CODE[precision], 3, put(ctx, w), put(ctx, x, precision), None, y, y1, rows, cols, m, 4 * group, 4 * group, last, 2, group)
    got = y.download(np.float32, (m, 4 * group))
    for n in range(4):
        assert worst(got[:, n * group:(n + 1) * group], x[n] @ w[n * group:(n + 1) * group].T.astype(np.float64)) < 1e-4, n
    want = np.tanh(x[4] @ w[4 * group:].T.astype(np.float64))
    assert np.all(np.abs(take(y1, (m, last), precision) - want) <= (1e-4 if precision == "float32" else 1 / 200) * (np.abs(want) + 0.05))


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("m,experts,top,ff,width,skew", [(2, 3, 1, 33, 70, 0.0), (65, 5, 2, 64, 128, 0.0), (300, 40, 4, 100, 192, 0.0), (130, 6, 3, 64, 96, 8.0), (512, 4, 4, 128, 256, 0.0),
                                                         (600, 8, 2, 192, 320, 3.0)])
def test_experts_of_a_chunk(ctx, m, experts, top, ff, width, skew, precision):
    """skew: one expert that most tokens choose, another that hardly any does."""
    g = np.random.default_rng(m + experts)
    ld, fp = pad_to(width), pad_to(ff)
    gate, up = cases.round_bf16(2 * g.standard_normal((2, experts, ff, width)) / np.sqrt(width))
    down, h = cases.round_bf16(g.standard_normal((experts, width, ff)) / np.sqrt(ff)), seen_as(g.standard_normal((m, width)), precision)
    logits = g.standard_normal((m, experts)).astype(np.float32)
    logits[:, 0] += skew
    logits[:, -1] -= skew
    pairs, dn = np.zeros((experts, fp, 2, ld), np.float32), np.zeros((experts, width, fp), np.float32)
    pairs[:, :ff, 0, :width], pairs[:, :ff, 1, :width], dn[:, :, :ff] = gate, up, down
    n, es = m * top, 4 if precision == "float32" else 2
    bufs = {"logits": f32(ctx, logits), "h": put(ctx, padded(h, m, ld), precision), "up": put(ctx, pairs), "down": put(ctx, dn), "chosen": ctx.alloc(n * 8), "place": ctx.alloc(n * 4),
            "table": ctx.alloc((1 + experts + n) * 16), "permuted": ctx.alloc(n * ld * es), "inner": ctx.alloc(n * fp * es), "rows": ctx.alloc(n * ld * 4).fill(0), "y": f32(ctx, np.full((m, ld), 5.0))}
    a = capi.MoeArgs(m=m, experts=experts, top=top, ff=ff, width=width, limit=1.0, **{k: b.ptr for k, b in bufs.items()})
    ctx.call("moe_rows", CODE[precision], C.byref(a), 5, 0)
    chosen = bufs["chosen"].download(np.int32, (m, top, 2))
    want_e, want_w = ref.route(logits.astype(np.float64), np.eye(experts), 0.0, top)
    np.testing.assert_array_equal(chosen[..., 0], want_e)
    assert worst(chosen[..., 1].copy().view(np.float32), want_w) < 1e-6
    place = bufs["place"].download(np.int32, (m, top))
    assert sorted(place.reshape(-1).tolist()) == list(range(n))
    assert all((np.diff(want_e.reshape(-1)[np.argsort(place.reshape(-1))]) >= 0))  # an expert's rows are neighbours
    want = np.zeros((m, width))
    for e in range(experts):
        at = np.argwhere(want_e == e)
        if len(at):
            want[at[:, 0]] += want_w[at[:, 0], at[:, 1]][:, None] * ref.expert(h[at[:, 0]], gate[e], up[e], down[e], 1.0)
    got = bufs["y"].download(np.float32, (m, ld))[:, :width]
    assert (worst if precision == "float32" else worst_row)(got, want) < (1e-4 if precision == "float32" else 0.01)
    assert ctx.device_error_flags() == 0
    for b in bufs.values():
        b.free()


# ── row kernels ─────────────────────────────────────────────────────────────
def test_embedding(ctx):
    g = np.random.default_rng(3)
    table, toks = cases.round_bf16(g.standard_normal((50, 70))), np.array([49, 0, 7], np.int32)
    x = f32(ctx, np.zeros((3, 128)))
    ctx.call("embed_rows", put(ctx, table), ctx.to_device(toks), x, 70, 128, 3, 50, 1.75)
    got = x.download(np.float32, (3, 128))
    np.testing.assert_allclose(got[:, :70], ref.embed(table, toks, 1.75), rtol=1e-6)
    assert not got[:, 70:].any()


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("width", [64, 70, 1500, 4096, 5000, 9000])
def test_residual_and_norms(ctx, width, precision):
    g = np.random.default_rng(width)
    m, ld = 5, pad_to(width)
    x, y = g.standard_normal((m, width)), 3 * g.standard_normal((m, width))
    post, norm = cases.round_bf16(0.4 * g.standard_normal((2, width)))
    dp, dn, out, h = put(ctx, padded(post, ld)), put(ctx, padded(norm, ld)), put(ctx, np.zeros((m, ld)), precision), f32(ctx, np.zeros((m, ld)))
    tol = EXACT if precision == "float32" else 0.04
    total = x + ref.zero_centred_norm(y, post, 1e-3)
    for rows in (None, np.array([3, 0, 3], np.int32)):
        dx, n = f32(ctx, padded(x, m, ld)), m if rows is None else len(rows)
        ctx.call("residual_norm_rows", CODE[precision], dx, f32(ctx, padded(y, m, ld)), dp, dn, None if rows is None else ctx.to_device(rows), out, h, width, ld, n, 1e-3)
        want = ref.zero_centred_norm(total if rows is None else total[rows], norm, 1e-3)
        assert worst(take(out, (m, ld), precision)[:n, :width], want) < tol and worst(h.download(np.float32, (m, ld))[:n, :width], want) < EXACT
        assert worst(dx.download(np.float32, (m, ld))[:, :width], total if rows is None else x) < EXACT
    dx = f32(ctx, padded(x, m, ld))
    ctx.call("residual_norm_rows", CODE[precision], dx, None, None, dn, None, out, None, width, ld, m, 1e-3)
    assert worst(take(out, (m, ld), precision)[:, :width], ref.zero_centred_norm(x, norm, 1e-3)) < tol


# ── latent attention ────────────────────────────────────────────────────────
class Latent:
    """One layer's cache on the device, fed portions of projections; want() follows with the restatement on
    what the cache holds (rounded to its type).  kind: how a portion of several rows is attended to."""

    def __init__(self, ctx, precision, heads, dim, rot, vdim, rank, window, scale, rot_dims=None, q_rank=20, chunk=64, base=500.0, seed=0):
        g = np.random.default_rng(seed)
        self.ctx, self.precision, self.H, self.dim, self.rot, self.vdim, self.rank, self.window, self.scale = ctx, precision, heads, dim, rot, vdim, rank, window, scale
        self.rot_dims, self.q_rank, self.base = rot if rot_dims is None else rot_dims, q_rank, base
        self.dp, self.rp, self.vp, self.kr, self.qp = pad_to(dim, 16), pad_to(rot, 16), row_elems(vdim), pad_to(rank), pad_to(q_rank)
        self.ring, self.es = pad_to(window + chunk), 4 if precision == "float32" else 2
        self.uk, self.uv = cases.round_bf16(g.standard_normal((heads, dim, rank)) / np.sqrt(rank)), cases.round_bf16(g.standard_normal((heads, vdim, rank)) / np.sqrt(rank))
        self.kv_norm, self.q_norm = cases.round_bf16(1 + 0.2 * g.standard_normal(rank)), cases.round_bf16(1 + 0.2 * g.standard_normal(q_rank))
        kv = np.concatenate([padded(self.uk, heads, self.dp, self.kr).reshape(-1, self.kr), padded(self.uv, heads, self.vp, self.kr).reshape(-1, self.kr)])
        self.kv_proj = put(ctx, kv)
        self.bufs = {"kv_proj": self.kv_proj, "kv_norm": put(ctx, self.kv_norm), "q_norm": put(ctx, padded(self.q_norm, self.qp)),
                     "rot_freq": ctx.to_device(base ** (-2.0 * np.arange(max(1, self.rot_dims // 2)) / max(1, self.rot_dims))),
                     "latent_ring": ctx.alloc(self.ring * self.kr * self.es).fill(0), "rot_ring": ctx.alloc(self.ring * self.rp * self.es).fill(0)}
        self.reset()

    def reset(self):
        self.n, self.c, self.kp = 0, np.zeros((0, self.rank)), np.zeros((0, self.rot))

    def feed(self, u, q, expand=True):
        """u [m, rank + rot] latent and key part projections, q [m, H, dim + rot]: z [m, H, vdim]."""
        ctx, m, H, first = self.ctx, len(u), self.H, self.n
        decode = m == 1
        act = "float32" if decode else self.precision
        ldu = self.qp + self.rank + self.rot
        qlat = np.random.default_rng(7).standard_normal((m, self.q_rank))
        rows = np.concatenate([padded(qlat, m, self.qp), u], 1)
        qrow = np.concatenate([padded(q[..., :self.dim], m, H, self.dp), padded(q[..., self.dim:], m, H, self.rp)], -1)
        bufs = {**self.bufs, "u": f32(ctx, rows), "q": put(ctx, qrow, act), "query_latent": put(ctx, np.zeros((m, self.qp)), self.precision), "qa": f32(ctx, np.zeros((m, H, self.kr + self.rp))),
                "sums": f32(ctx, np.zeros((64 if decode else m) * H * self.kr)), "maxima": f32(ctx, np.zeros((64 if decode else m) * H * 2)), "z": put(ctx, np.full((m, H * self.vp + 2), 9.0), act)}
        a = capi.LatentArgs(heads=H, dim=self.dim, rot_dim=self.rot, rot_dims=self.rot_dims, vdim=self.vdim, kv_rank=self.rank, q_rank=self.q_rank, own=1, window=self.window, ring=self.ring,
                            scale=self.scale, eps=1e-4, m=m, ldu=ldu, ldz=H * self.vp + 2, decode=int(decode), **{k: b.ptr for k, b in bufs.items()})
        code = CODE[self.precision]
        if not decode:
            ctx.call("latent_append", code, C.byref(a), first)
            want = ref.plain_norm(qlat, self.q_norm, 1e-4)
            assert worst(take(bufs["query_latent"], (m, self.qp), self.precision)[:, :self.q_rank], want) < (EXACT if self.precision == "float32" else 0.02)
        tiled = not decode and expand and self.precision == "bfloat16" and self.dp + self.rp <= 320 and self.vp <= 256
        if tiled:
            live, n = min(self.ring, first + m), H * (self.dp + self.vp)
            kv_rows = ctx.alloc(self.ring * n * 2).fill(0)
            ctx.call("dense_gemm_ex", code, 2, self.kv_proj, self.bufs["latent_ring"], None, kv_rows, None, n, self.kr, live, n, n, 0, 0, 0)
            a.kv_rows = kv_rows.ptr
            ctx.call("latent_prefill", C.byref(a), first)
        else:
            for step in ("query", "scores", "values"):
                ctx.call("latent_" + step, code, C.byref(a), first)
        out = take(bufs["z"], (m, H * self.vp + 2), act)
        assert (out[:, H * self.vp:] == 9.0).all()
        self.remember(u, m)
        return out[:, :H * self.vp].reshape(m, H, self.vp)[..., :self.vdim]

    def remember(self, u, m):
        pos = self.n + np.arange(m)
        self.c = np.concatenate([self.c, seen_as(ref.plain_norm(u[:, :self.rank], self.kv_norm, 1e-4), self.precision)])
        self.kp = np.concatenate([self.kp, seen_as(ref.rotate_interleaved(u[:, self.rank:], pos, self.base, self.rot_dims), self.precision)])
        self.n += m

    def want(self, q):
        """Of all positions so far."""
        qr = ref.rotate_interleaved(q[..., self.dim:], range(self.n), self.base, self.rot_dims)
        return ref.latent_window_attention(q[..., :self.dim], qr, self.c, self.kp, self.uk.astype(np.float64), self.uv.astype(np.float64), 0, self.scale, self.window)

    def inputs(self, n, seed=1):
        g = np.random.default_rng(seed)
        return g.standard_normal((n, self.rank + self.rot)), seen_as(g.standard_normal((n, self.H, self.dim + self.rot)), self.precision)

    def run(self, u, q, cuts, expand=True):
        out, at = [], 0
        for c in cuts:
            out.append(self.feed(u[at:at + c], q[at:at + c], expand))
            at += c
        return np.concatenate(out)


GEOMETRIES = [dict(heads=4, dim=32, rot=16, vdim=48, rank=40, window=24, scale=0.2), dict(heads=17, dim=20, rot=6, vdim=18, rank=33, window=1, scale=0.3),
              dict(heads=1, dim=70, rot=34, vdim=100, rank=130, window=45, scale=0.1), dict(heads=16, dim=128, rot=64, vdim=128, rank=512, window=200, scale=0.07),
              dict(heads=33, dim=16, rot=8, vdim=256, rank=64, window=90, scale=0.25), dict(heads=2, dim=64, rot=32, vdim=130, rank=520, window=70, scale=0.1),
              dict(heads=2, dim=300, rot=40, vdim=300, rank=64, window=33, scale=0.06), dict(heads=3, dim=16, rot=20, vdim=16, rank=16, window=40, scale=0.3, rot_dims=8)]
ATTENTION_LIMIT = {"float32": 1e-4, "bfloat16": 0.03}


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("case", range(len(GEOMETRIES)))
def test_latent_attention(ctx, case, precision):
    a = Latent(ctx, precision, **GEOMETRIES[case])
    n = 170
    u, q = a.inputs(n)
    for cuts, expand in (([64, 64, 42], True), ([2, 5, 30, 1, 1, 64, 2, 3, 62], True), ([50] + [1] * 40 + [60, 20], True), ([3, 64, 1, 64, 38], False)):
        a.reset()
        got = a.run(u, q, cuts, expand)
        assert worst_row(got, a.want(q)) < ATTENTION_LIMIT[precision], (cuts, expand)


@pytest.mark.parametrize("precision", PRECISIONS)
def test_last_key_of_the_window_and_the_one_before(ctx, precision):
    """One key stands out for every query: seen while it is window - 1 tokens back, not one later; at a
    ring's end, a tile's edge and the sequence's start; in prompts, portions and decoded tokens."""
    geometry = dict(heads=2, dim=16, rot=16, vdim=16, rank=16, window=40, scale=1.0, base=1e6)
    for special in (0, 1, 31, 63, 64, 100, 103, 104, 127):
        a = Latent(ctx, precision, **geometry)
        u, q = a.inputs(210, seed=special)
        u *= 0.05
        u[:, :16] += 1.0  # every latent alike, so every value alike
        u[special, :16] = -1.0
        q[..., :16] = seen_as(-6.0 * (a.uk.astype(np.float64) @ (np.ones(16) * a.kv_norm))[None] / 3, precision)  # unrotated queries that point at the odd latent's key
        q[..., 16:] = 0
        for cuts in ([64, 64, 64, 18], [64, 30] + [1] * 100 + [16], [7, 2, 64, 11, 2, 2, 2, 64, 2, 56]):
            a.reset()
            got = a.run(u, q, cuts)
            want = a.want(q)
            assert worst_row(got, want) < ATTENTION_LIMIT[precision]
            far = np.abs(want[special + 39] - want[special + 40]).max() / np.abs(want).max()
            assert far > 0.1, special  # the edge shows


@pytest.mark.parametrize("precision", PRECISIONS)
def test_rows_used_again_are_not_seen(ctx, precision):
    """A second sequence over what the first left, which would swamp every softmax if it were seen."""
    a = Latent(ctx, precision, heads=4, dim=32, rot=16, vdim=48, rank=40, window=24, scale=0.2)
    u, q = a.inputs(150, seed=5)
    a.run(30 * u, q, [64, 64, 22])
    a.reset()
    u, q = a.inputs(100, seed=6)
    assert worst_row(a.run(u, q, [1, 2, 40, 1, 1, 55]), a.want(q)) < ATTENTION_LIMIT[precision]


def test_far_positions_keep_exact_angles(ctx):
    """Scores depend on how far apart tokens are, also a million positions on."""
    a = Latent(ctx, "float32", heads=2, dim=16, rot=32, vdim=16, rank=16, window=30, scale=0.3, base=20.0)
    u, q = a.inputs(40, seed=3)
    near = a.run(u, q, [40])
    a.reset()
    a.n = 1_000_003
    at, out = 0, []
    for c in (20, 1, 19):
        out.append(a.feed(u[at:at + c], q[at:at + c]))
        at += c
    # the first rows' windows reach back to rows that were never written
    assert worst(np.concatenate(out)[30:], near[30:]) < 2e-4


# ── time mixing ─────────────────────────────────────────────────────────────
class TimeMix:
    """State on the device, fed portions of projections."""

    def __init__(self, ctx, precision, heads, dim, rank, width, seed=0):
        g = np.random.default_rng(seed)
        self.ctx, self.precision, self.H, self.D, self.width = ctx, precision, heads, dim, width
        self.n, self.group, self.rp, self.ld = heads * dim, pad_to(heads * dim, 128), pad_to(rank), pad_to(width)
        self.w2, self.w0 = cases.round_bf16(g.standard_normal((self.n, rank)) / np.sqrt(rank)), cases.round_bf16(g.uniform(-4, 0.5, self.n))
        self.bonus, self.norm, self.mu = cases.round_bf16(g.standard_normal((heads, dim))), cases.round_bf16(1 + 0.2 * g.standard_normal(self.n)), cases.round_bf16(g.uniform(0, 1, (5, width)))
        self.bufs = {"w2": put(ctx, padded(self.w2, self.n, self.rp)), "w0": put(ctx, self.w0), "bonus": put(ctx, self.bonus), "norm": put(ctx, self.norm), "mu": put(ctx, padded(self.mu, 5, self.ld)),
                     "state": ctx.alloc(heads * dim * dim * 4).fill(0x7F), "before": ctx.alloc(self.ld * 4).fill(0x7F)}  # position 0 reads neither
        self.position = 0

    def feed(self, p, inner, h):
        """p [4, m, n] projections r, k, v, g; inner [m, rank]; h [m, width]: (z [m, n], mixes [5, m, width] or None)."""
        ctx, m = self.ctx, p.shape[1]
        rows = np.concatenate([padded(x, m, self.group) for x in p], 1)
        act = "float32" if m == 1 else self.precision
        es = 4 if act == "float32" else 2
        ldz = pad_to(self.n)
        if m == 1:
            rows = np.concatenate([rows, padded(inner, 1, self.rp)], 1)
        z, hd = put(ctx, np.zeros((m, ldz)), act), f32(ctx, padded(h, m, self.ld))
        a = capi.WkvArgs(heads=self.H, dim=self.D, rank=self.rp, ld=self.ld, m=m, ldu=rows.shape[1], ldz=ldz, eps=1e-4, **{k: b.ptr for k, b in {**self.bufs, "u": f32(ctx, rows), "h": hd}.items()})
        keep, mixes = [], None
        if m == 1:
            a.out = z.ptr
            u = f32(ctx, rows)
            a.u = u.ptr
            ctx.call("wkv_decode", C.byref(a), self.position)
        else:
            code = CODE[self.precision]
            out, o, u = ctx.alloc(5 * m * self.ld * es), f32(ctx, np.zeros((m, self.n))), f32(ctx, rows)
            decay = f32(ctx, np.exp(-np.exp(np.tanh(inner) @ self.w2.T.astype(np.float64) + self.w0)))
            a.u, a.out = u.ptr, out.ptr
            ctx.call("wkv_shift", code, C.byref(a), self.position)
            mixes = take(out, (5, m, self.ld), self.precision)[..., :self.width]
            a.decay, a.out = decay.ptr, o.ptr
            ctx.call("wkv_prefill", C.byref(a), self.position)
            a.o, a.out = o.ptr, z.ptr
            ctx.call("wkv_gate", code, C.byref(a))
            keep += [out, o, u, decay]
        self.position += m
        return take(z, (m, ldz), act)[:, :self.n], mixes

    def want(self, p, inner):
        T = p.shape[1]
        r, k, v = (x.reshape(T, self.H, self.D) for x in p[:3])
        w = np.exp(-np.exp(np.tanh(inner) @ self.w2.T.astype(np.float64) + self.w0)).reshape(T, self.H, self.D)
        o, state = ref.wkv(r, k, v, w, self.bonus.astype(np.float64), np.zeros((self.H, self.D, self.D)))
        return ref.unit_rms(o, 1e-4).reshape(T, -1) * self.norm * ref.silu(p[3]), state


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("heads,dim,rank,width", [(3, 32, 24, 96), (2, 33, 7, 70), (1, 64, 64, 64), (5, 16, 70, 320), (2, 128, 130, 200), (1, 200, 24, 96), (1, 256, 200, 64), (3, 10, 5, 33), (4, 72, 64, 128)])
def test_time_mixing(ctx, heads, dim, rank, width, precision):
    t = TimeMix(ctx, precision, heads, dim, rank, width)
    g = np.random.default_rng(dim)
    n = 90
    p, inner, h = g.standard_normal((4, n, heads * dim)).astype(np.float32).astype(np.float64), g.standard_normal((n, rank)).astype(np.float32).astype(np.float64), g.standard_normal((n, width))
    want, state = t.want(p, inner)
    tol = 1e-4 if precision == "float32" else 0.01
    for cuts in ([n], [1] * 20 + [n - 20], [2, 3, 1, 16, 17, 1, 30, 1, n - 71], [n - 9] + [1] * 9):
        t.position, at = 0, 0
        for c in cuts:
            z, mixes = t.feed(p[:, at:at + c], inner[at:at + c], h[at:at + c])
            assert worst_row(z, want[at:at + c]) < tol * (np.sqrt(np.mean(want ** 2)) / np.sqrt(np.mean(want[at:at + c] ** 2))), (cuts[:4], at)
            if mixes is not None:
                shifted = ref.token_shift(h[at:at + c], h[at - 1] if at else np.zeros(width))
                for s in range(5):
                    assert worst(mixes[s], ref.mixed(h[at:at + c], shifted, t.mu[s])) < (1e-5 if precision == "float32" else 0.02)
            at += c
        got = t.bufs["state"].download(np.float32, (heads, dim, dim))
        assert worst(got, state) < 1e-4, cuts[:4]
        assert worst(t.bufs["before"].download(np.float32, t.ld)[:width], h[-1]) < 1e-6


def test_a_decay_that_hardly_decays_carries_the_first_token(ctx):
    """Far back: only the first token has a key, and the last ones still read it."""
    t = TimeMix(ctx, "float32", 2, 32, 8, 64)
    t.w0[:] = -12.0
    t.w2[:] = 0
    t.bufs["w0"], t.bufs["w2"] = put(ctx, t.w0), put(ctx, padded(t.w2, t.n, t.rp))
    g = np.random.default_rng(1)
    n = 700
    p = g.standard_normal((4, n, 64)).astype(np.float32).astype(np.float64)
    p[1, 1:] = 0
    p[0] = p[1, :1] + 0.3 * p[0]  # every query near the one key
    want, _ = t.want(p, np.zeros((n, 8)))
    z = np.concatenate([t.feed(p[:, a:b], np.zeros((b - a, 8)), np.zeros((b - a, 64)))[0] for a, b in ((0, 300), (300, 301), (301, 700))])
    assert worst(z, want) < 1e-4 and np.abs(want[-1]).max() > 0.1


# ── whole models ────────────────────────────────────────────────────────────
def open_decoder(ctx, name, precision, max_chunk=64, **kw):
    cfg = cases.ALL[name]
    t = cases.tensors(cfg)
    arch = checkpoint.architecture(cfg)
    return arch.decoder(ctx, arch.parse(cfg), checkpoint.TensorFile(cases.stored(t)), precision=precision, max_chunk=max_chunk, **kw), ref.Kesedra(cfg, t)


LIMIT = {"float32": 2e-5, "bfloat16": 0.04}  # of worst_row
_reference = {}


def reference_logits(name, m, toks):
    key = (name, tuple(toks.tolist()))
    if key not in _reference:
        m.reset()
        _reference[key] = m.feed(toks)
    return _reference[key]


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("name", cases.ALL)
def test_model_whole_portions_and_decoded(ctx, name, precision):
    dec, m = open_decoder(ctx, name, precision)
    n = 150
    toks = cases.tokens(cases.ALL[name], n)
    want = reference_logits(name, m, toks)
    for cuts in ([n], [2] * 10 + [n - 20], [3, 17, 1, 1, 50, 2, 33, 1, 1, 1, n - 110], [n - 80] + [1] * 80, [1] * n):
        err = worst_row(run_cuts(dec, toks, cuts), want)
        assert err < LIMIT[precision], (cuts[:6], err)


@pytest.mark.parametrize("precision", PRECISIONS)
def test_cache_and_state_are_used_again_without_clearing(ctx, precision):
    dec, m = open_decoder(ctx, "mixed", precision)
    for n, seed, cuts in ((140, 3, [139, 1]), (1, 4, [1]), (23, 5, [2, 21]), (90, 6, [60] + [1] * 30), (140, 3, [1] * 20 + [120])):
        toks = cases.tokens(cases.MIXED, n, seed)
        assert worst_row(run_cuts(dec, toks, cuts), reference_logits("mixed", m, toks)) < LIMIT[precision]


def test_mistakes_in_the_restatement_show(ctx):
    """Planted there: a window one longer, a bonus that stays in the state, a cut state, a router without weights, a rotation of halves."""
    dec, m = open_decoder(ctx, "mixed", "float32")
    toks = cases.tokens(cases.MIXED, 120, 9)
    got = dec.feed(toks, 0, range(120))
    want = reference_logits("mixed", m, toks)
    assert worst_row(got, want) < LIMIT["float32"]
    kept = {n: getattr(ref, n) for n in ("window_positions", "wkv", "token_shift", "route", "rotate_interleaved", "silu")}

    def lasting_bonus(r, k, v, w, u, state):
        o, s = kept["wkv"](r, k, v, w, u, state)
        return o, s + u[..., None] * 1e-2

    def even_weights(h, router, bias, top):
        chosen, weights = kept["route"](h, router, bias, top)
        return chosen, np.full_like(weights, 1 / top)

    def halves(x, positions, base, dims):
        order = np.arange(dims).reshape(2, -1).T.reshape(-1)  # pairs (i, i + dims / 2)
        out = np.array(x, np.float64)
        out[..., order] = kept["rotate_interleaved"](x[..., order], positions, base, dims)
        return out
    planted = {"window_positions": lambda i, s: kept["window_positions"](i, s + 1), "wkv": lasting_bonus, "token_shift": lambda h, b: kept["token_shift"](h, 0 * b), "route": even_weights,
               "rotate_interleaved": halves, "silu": lambda z: np.maximum(z, 0)}
    for name, fn in planted.items():
        try:
            setattr(ref, name, fn)
            m.reset()
            wrong = np.concatenate([m.feed(toks[:60]), m.feed(toks[60:])])
        finally:
            setattr(ref, name, kept[name])
        assert worst_row(got, wrong) > 50 * LIMIT["float32"], name


def test_only_wanted_rows(ctx):
    dec, m = open_decoder(ctx, "odd", "float32", max_chunk=32, capacity=640)
    toks = cases.tokens(cases.ODD, 90)
    want = reference_logits("odd", m, toks)
    places = [64, 3, 89, 31, 32, 3]
    assert worst(dec.feed(toks, 0, places), want[places]) < 1e-4
    assert dec.feed(toks[:1], 0, []).shape == (0, 97)
    with pytest.raises(ValueError):
        dec.feed(toks[:4], 0, [4])
    with pytest.raises(capi.SmeltError):
        dec.feed([97, 1], 0, [0])  # an id past the vocabulary
    with pytest.raises(capi.SmeltError):
        dec.feed(toks[:2], 639, [0])  # positions past the capacity asked for


@pytest.mark.parametrize("use_graph", [True, False])
def test_greedy_generation(ctx, use_graph):
    dec, m = open_decoder(ctx, "mixed", "float32")
    prompt = cases.tokens(cases.MIXED, 70, 8)
    got = dec.generate(prompt, 60, use_graph=use_graph)[:, 0]
    m.reset()
    logits = m.feed(np.concatenate([prompt, got[:-1]]))[len(prompt) - 1:]
    top = np.sort(logits, 1)[:, ::-1]
    clear = top[:, 0] - top[:, 1] > 1e-3 * logits.std()
    assert clear.sum() > 50
    np.testing.assert_array_equal(got[clear], logits.argmax(1)[clear])


def test_long_decoding(ctx):
    """Several times round every ring, through the graph's multi-token replay."""
    dec, m = open_decoder(ctx, "odd", "float32", max_chunk=16)
    prompt = cases.tokens(cases.ODD, 9, 12)
    got = dec.generate(prompt, 400)[:, 0]
    toks = np.concatenate([prompt, got])
    m.reset()
    logits = m.feed(toks[:-1])
    clear = np.diff(np.sort(logits, 1)[:, -2:], axis=1)[:, 0] > 1e-3 * logits.std()
    np.testing.assert_array_equal(toks[1:][8:][clear[8:]], logits.argmax(1)[8:][clear[8:]])
    assert worst(run_cuts(dec, toks[:-1], [300] + [1] * 108)[-1:], logits[-1:]) < 1e-3


def test_table_step_equals_graph_step(ctx):
    dec, _ = open_decoder(ctx, "mixed", "bfloat16")
    toks = cases.tokens(cases.MIXED, 40, 2)
    eager = []
    for i, t in enumerate(toks):
        dec.decode_step([t], i)
        eager.append(dec.logits(1)[0])
    np.testing.assert_array_equal(run_cuts(dec, toks, [1] * 40), np.stack(eager))


def test_snapshot_restores_cache_and_state(ctx):
    dec, _ = open_decoder(ctx, "mixed", "bfloat16")
    toks = cases.tokens(cases.MIXED, 120, 3)
    dec.feed(toks[:100], 0, [])
    snap = dec.capture_snapshot(100)
    first = run_cuts_from(dec, toks, 100)
    dec.feed(cases.tokens(cases.MIXED, 120, 4), 0, [])
    dec.restore_snapshot(snap)
    np.testing.assert_array_equal(run_cuts_from(dec, toks, 100), first)
    snap.close()


@pytest.mark.parametrize("precision", PRECISIONS)
def test_trace_run_program(ctx, tmp_path, precision):
    cfg, t = cases.MIXED, cases.tensors(cases.MIXED)
    model, out = tmp_path / "model", tmp_path / "out"
    model.mkdir(), out.mkdir()
    (model / "config.json").write_text(json.dumps(cfg))
    checkpoint.write_safetensors(str(model / "model.safetensors"), cases.stored(t))
    a, b = cases.tokens(cfg, 100, 5), cases.tokens(cfg, 30, 6)
    steps = [([("a", a[:77], [0, 76])], []), ([("a", a[77:98], [20])], []), ([("a", a[98:99], [])], []), ([("a", a[99:], [0])], ["a"]), ([("b", b, [29])], ["b"])]
    lines = "".join(json.dumps({"step": i, "entries": [{"id": n, "tokens": x.tolist(), "want": w} for n, x, w in e], "end": end}) + "\n" for i, (e, end) in enumerate(steps))
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", precision, "--out", str(out), "--max-tokens", "100"], input=lines,
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.split("\n") if x] == [f"done {i}" for i in range(5)]
    m = ref.Kesedra(cfg, t)
    la = m.feed(a)
    m.reset()
    lb = m.feed(b)
    read = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
    for i, want in ((0, la[[0, 76]]), (1, la[[97]]), (3, la[[99]]), (4, lb[[29]])):
        assert worst_row(read(i), want) < LIMIT[precision]
    assert not (out / "2.f32").exists()


@pytest.mark.parametrize("precision", PRECISIONS)
def test_package_runs_as_the_model_does(ctx, tmp_path, precision):
    cfg = cases.MIXED
    arch, t = checkpoint.architecture(cfg), cases.tensors(cfg)
    arch.write_package(str(tmp_path / "m.smeltpkg"), arch.parse(cfg), checkpoint.TensorFile(cases.stored(t)), precision=precision, max_chunk=64)
    dec, _ = open_decoder(ctx, "mixed", precision)
    prompt = cases.tokens(cfg, 90, 21)
    want = dec.generate(prompt, 30)[:, 0]
    other = capi.Context(0)
    session = package.PackageSession(other, str(tmp_path / "m.smeltpkg"))
    got = [session.prefill(prompt, chunk=64)]
    for i in range(9):
        got.append(session.decode_step(got[-1], 90 + i))
    session.build_graph()
    for i in range(9, 29):
        got.append(session.graph_step(got[-1], 90 + i))
    np.testing.assert_array_equal(got, want)
    with pytest.raises(capi.SmeltError):
        session.prefill(prompt, chunk=90)  # more than the tables were compiled for
    other.close()


def test_generate_command(tmp_path, capsys, ctx):
    from smelt_b200 import generate

    cfg = cases.ODD
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    checkpoint.write_safetensors(str(tmp_path / "model.safetensors"), cases.stored(cases.tensors(cfg)))
    dec, _ = open_decoder(ctx, "odd", "float32")
    assert generate.main(["--model", str(tmp_path), "--prompt", "5,6,7,8", "--tokens", "12", "--dtype", "float32"]) == 0
    assert [int(x) for x in capsys.readouterr().out.split()] == dec.generate([5, 6, 7, 8], 12)[:, 0].tolist()
