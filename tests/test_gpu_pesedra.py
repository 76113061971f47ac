"""Pesedra on the GPU against the float64 restatement: each kernel alone, then whole models through the
framework's loader, tables, graph and trace replay."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import pesedra_cases as cases
from oracle import pesedra as ref
from smelt_b200 import capi, checkpoint, package, pesedra

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PRECISIONS = ["bfloat16", "float32"]


@pytest.fixture(scope="module")
def ctx():
    c = capi.Context(0)
    yield c
    assert c.device_error_flags() == 0
    c.close()


def pad_to(n, k=64):
    return -(-n // k) * k


def row_elems(d):
    return 64 if d <= 64 else 128 if d <= 128 else 256 if d <= 256 else pad_to(d)


def put(ctx, a, precision="bfloat16"):
    """A device copy in the activations' type."""
    a = np.ascontiguousarray(a, np.float32)
    return ctx.to_device(a if precision == "float32" else checkpoint.f32_to_bf16(a))


def take(buf, shape, precision):
    return buf.download(np.float32, shape) if precision == "float32" else checkpoint.bf16_to_f32(buf.download(np.uint16, shape)).reshape(shape)


def seen_as(a, precision):
    """The values the device holds after storing a in the activations' type."""
    return np.asarray(a, np.float32).astype(np.float64) if precision == "float32" else cases.round_bf16(a).astype(np.float64)


def worst(got, want):
    """Largest difference over the reference's root mean square."""
    want = np.asarray(want, np.float64)
    return float(np.max(np.abs(got - want)) / np.sqrt(np.mean(want * want)))


def worst_row(got, want):
    """The same for the root-mean-square difference of a row (the last axis): the measure for 16-bit outputs."""
    want = np.asarray(want, np.float64)
    return float(np.max(np.sqrt(np.mean((got - want) ** 2, -1))) / np.sqrt(np.mean(want * want)))


# ── projections ─────────────────────────────────────────────────────────────
GEMM_SHAPES = [(7, 64, 1), (130, 64, 2), (320, 192, 17), (300, 1024, 65), (200, 4096, 33), (1024, 2048, 300), (5000, 128, 130), (96, 8192, 16), (257, 320, 513)]


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("rows,cols,m", GEMM_SHAPES)
def test_dense_gemm(ctx, rows, cols, m, precision):
    g = np.random.default_rng(rows + cols + m)
    code = package.DenseDecoder.PRECISIONS[precision]
    w, x = cases.round_bf16(g.standard_normal((rows, cols)) / np.sqrt(cols)), seen_as(g.standard_normal((m, cols)), precision)
    want = x @ w.T.astype(np.float64)
    dw, dx = put(ctx, w), put(ctx, x, precision)
    tol = 1e-4
    ld = rows + 3
    y = put(ctx, np.full((m, ld), 7.0), "float32")
    ctx.call("dense_gemm", code, 0, dw, dx, y, None, rows, cols, m, rows, ld, 0, 0.0, 0.0)
    got = y.download(np.float32, (m, ld))
    assert worst(got[:, :rows], want) < tol and (got[:, rows:] == 7.0).all()
    ctx.call("dense_gemm", code, 1, dw, dx, y, None, rows, cols, m, rows, ld, 0, 0.0, 0.0)
    assert worst(y.download(np.float32, (m, ld))[:, :rows], 2 * want) < tol
    # the first rows stored, the rest through xIELU
    split, rising, falling = rows // 3, 0.8, 1.1
    y0, y1 = put(ctx, np.zeros((m, split + 1)), precision), put(ctx, np.full((m, rows), 5.0), precision)
    ctx.call("dense_gemm", code, 2, dw, dx, y0, y1, rows, cols, m, split, split + 1, rows, rising, falling)
    rest = want[:, split:]
    neg = np.minimum(rest, 0)
    act = np.where(rest > 0, rising * rest * rest, falling * (np.expm1(neg) - neg)) + rest / 2
    out_tol = 1e-4 if precision == "float32" else 1.0 / 256
    lhs, rhs = take(y0, (m, split + 1), precision), take(y1, (m, rows), precision)
    assert np.all(np.abs(lhs[:, :split] - want[:, :split]) <= out_tol * (np.abs(want[:, :split]) + 0.05))
    assert np.all(np.abs(rhs[:, :rows - split] - act) <= out_tol * (np.abs(act) + 0.05)) and (rhs[:, rows - split:] == 5.0).all()
    assert ctx.device_error_flags() == 0
    for b in (dw, dx, y, y0, y1):
        b.free()


@pytest.mark.parametrize("rows,cols", [(1, 64), (3, 128), (37, 320), (1000, 4096), (4099, 192), (130, 16384), (20000, 256)])
def test_dense_matvec(ctx, rows, cols):
    g = np.random.default_rng(rows * 7 + cols)
    w, x = cases.round_bf16(g.standard_normal((rows, cols)) / np.sqrt(cols)), g.standard_normal(cols).astype(np.float32)
    want = w.astype(np.float64) @ x.astype(np.float64)
    dw, dx = put(ctx, w), put(ctx, x, "float32")
    y, y1 = put(ctx, np.zeros(rows), "float32"), put(ctx, np.zeros(rows), "float32")
    ctx.call("dense_matvec", 0, dw, dx, None, 0, y, None, rows, cols, rows, 0, 0.0, 0.0, 0.0, 0.0)
    assert worst(y.download(np.float32, rows), want) < 3e-5
    ctx.call("dense_matvec", 1, dw, dx, None, 0, y, None, rows, cols, rows, 0, 0.0, 0.0, 0.0, 0.0)
    assert worst(y.download(np.float32, rows), 2 * want) < 3e-5
    # two source rows, the norm's factor, and the split with xIELU
    ka, split = cols // 2, rows // 2
    xa, xb = put(ctx, x[:ka], "float32"), put(ctx, x[ka:], "float32")
    f = 0.6 / np.sqrt(np.sum(x.astype(np.float64) ** 2) / (cols - 5) + 1e-3)
    ctx.call("dense_matvec", 0, dw, xa, xb, ka, y, y1, rows, cols, split, cols - 5, 0.6, 1e-3, 0.7, 1.3)
    got, rest = y.download(np.float32, rows), want[split:] * f
    neg = np.minimum(rest, 0)
    act = np.where(rest > 0, 0.7 * rest * rest, 1.3 * (np.expm1(neg) - neg)) + rest / 2
    if split:
        assert worst(got[:split], want[:split] * f) < 3e-5
    assert worst(y1.download(np.float32, rows - split), act) < 3e-5
    for b in (dw, dx, xa, xb, y, y1):
        b.free()


# ── row kernels ─────────────────────────────────────────────────────────────
def test_embedding_and_positions(ctx):
    g = np.random.default_rng(3)
    table, pos, toks, width, ld = cases.round_bf16(g.standard_normal((50, 70))), cases.round_bf16(g.standard_normal((40, 70))), np.array([49, 0, 7], np.int32), 70, 128
    x, x0 = put(ctx, np.zeros((3, ld)), "float32"), put(ctx, np.zeros((3, ld)), "float32")
    ctx.call("embed_positions", put(ctx, table), ctx.to_device(toks), put(ctx, pos), x, x0, width, ld, 3, 50, 40, 2.5, 37)
    want = np.zeros((3, ld))
    want[:, :70] = ref.embed(table, pos, toks, np.arange(37, 40), 2.5)
    for b in (x, x0):
        np.testing.assert_allclose(b.download(np.float32, (3, ld)), want, rtol=1e-6, atol=1e-6)
    assert ctx.call_status("embed_positions", x, x, x, x, x0, width, ld, 3, 50, 40, 2.5, 38) == capi.BAD_ARGUMENT  # past the table


@pytest.mark.parametrize("precision", PRECISIONS)
def test_scalar_norm_and_loop_pair(ctx, precision):
    g = np.random.default_rng(4)
    code = package.DenseDecoder.PRECISIONS[precision]
    x = np.zeros((9, 128), np.float32)
    x[:, :75] = g.standard_normal((9, 75)) * np.logspace(-3, 2, 9)[:, None]
    dx, tol = put(ctx, x, "float32"), 1e-6 if precision == "float32" else 1 / 256
    for rows in (None, [8, 0, 3, 3]):
        n = 9 if rows is None else 4
        out = put(ctx, np.zeros((n, 128)), precision)
        ctx.call("scalar_norm_rows", code, dx, None if rows is None else ctx.to_device(np.array(rows, np.int32)), out, 75, 128, n, -1.7, 1e-4)
        want = ref.scalar_rms_norm(x[:, :75].astype(np.float64), -1.7, 1e-4)[rows if rows is not None else slice(None)]
        np.testing.assert_allclose(take(out, (n, 128), precision)[:, :75], want, rtol=tol, atol=1e-7)
    x0 = g.standard_normal((9, 128)).astype(np.float32)
    out = put(ctx, np.zeros((9, 256)), precision)
    ctx.call("pair_rows", code, dx, put(ctx, x0, "float32"), out, 128, 9)
    np.testing.assert_array_equal(take(out, (9, 256), precision), seen_as(np.concatenate([x, x0], 1), precision))


# ── attention ───────────────────────────────────────────────────────────────
class Window:
    """One layer's cache on the device, fed with projections; chunks of one go through the decode kernel."""

    def __init__(self, ctx, precision, H, G, dim, vdim, window, pool, scale, softcap, positions, chunk, eps=1e-4, seed=0):
        self.ctx, self.precision, self.code = ctx, precision, package.DenseDecoder.PRECISIONS[precision]
        self.H, self.G, self.dim, self.vdim, self.kp, self.vp = H, G, dim, vdim, row_elems(dim), row_elems(vdim)
        ring = pad_to(max(window, pool) + chunk)
        self.desc = capi.WindowDesc(H, G, dim, vdim, window, pool, ring, positions // pool, scale, softcap, eps)
        es = 4 if precision == "float32" else 2
        rows = G * (ring + positions // pool)
        self.k, self.v = ctx.alloc(rows * self.kp * es).fill(0), ctx.alloc(rows * self.vp * es).fill(0)
        g = np.random.default_rng(seed)
        self.qn, self.kn = (cases.round_bf16(1 + 0.2 * g.standard_normal(dim)) for _ in "qk")
        self.dqn, self.dkn = put(ctx, self.qn), put(ctx, self.kn)
        self.at = 0

    def feed(self, u):
        m, ldz = len(u), pad_to(self.H * self.vdim)
        if m == 1:
            z, q = put(self.ctx, np.zeros(self.H * self.vdim), "float32"), self.ctx.alloc(self.H * self.kp * 4)
            self.ctx.call("window_decode", self.code, C.byref(self.desc), put(self.ctx, u, "float32"), self.dqn, self.dkn, self.k, self.v, q, z, self.at)
            out = z.download(np.float32, (1, self.H, self.vdim))
        else:
            q, z = put(self.ctx, np.zeros((m, self.H, self.kp)), self.precision), put(self.ctx, np.zeros((m, ldz)), self.precision)
            self.ctx.call("window_append", self.code, C.byref(self.desc), put(self.ctx, u, self.precision), self.dqn, self.dkn, self.k, self.v, q, m, self.at)
            self.ctx.call("window_pool", self.code, C.byref(self.desc), self.k, self.v, m, self.at)
            self.ctx.call("window_attention", self.code, C.byref(self.desc), q, self.k, self.v, z, ldz, m, self.at)
            full = take(z, (m, ldz), self.precision)
            assert not full[:, self.H * self.vdim:].any()
            out = full[:, :self.H * self.vdim].reshape(m, self.H, self.vdim)
        self.at += m
        return out

    def split(self, u):
        n, H, G, d, dv = len(u), self.H, self.G, self.dim, self.vdim
        return u[:, :H * d].reshape(n, H, d), u[:, H * d:(H + G) * d].reshape(n, G, d), u[:, (H + G) * d:].reshape(n, G, dv)

    def want(self, u, cuts=None):
        """The restatement on the values as the device stores them: a decoded token's projections stay fp32."""
        chunked = np.repeat([c > 1 for c in cuts or [len(u)]], cuts or [len(u)])[:, None]
        q, k, v = self.split(np.where(chunked, seen_as(u, self.precision), seen_as(u, "float32")))
        v = seen_as(v, self.precision)
        q, k = (seen_as(ref.head_rms_norm(x, w, self.desc.eps), self.precision) for x, w in ((q, self.qn), (k, self.kn)))
        d = self.desc
        if d.softcap <= 0:  # the restatement always caps; a huge cap is none
            return ref.window_pool_attention(q, k, v, 0, d.scale, 1e12, d.window, d.pool)
        return ref.window_pool_attention(q, k, v, 0, d.scale, d.softcap, d.window, d.pool)


GEOMETRIES = [  # H, G, dim, vdim, window, pool
    (4, 2, 64, 64, 40, 8), (8, 1, 128, 64, 33, 7), (5, 5, 48, 80, 16, 16), (12, 1, 64, 128, 100, 1), (20, 1, 32, 256, 24, 5), (4, 2, 256, 256, 64, 9),
    (3, 3, 300, 64, 20, 6), (4, 2, 64, 64, 5, 12), (2, 1, 33, 51, 1, 1), (9, 3, 128, 128, 130, 64), (18, 2, 96, 40, 48, 3)]
CUTS = [(2, 3, 1, 1, 37, 64, 1, 2, 64, 1, 9, 1, 1, 30), (64,) * 3 + (1,) * 24, (1,) * 5 + (40, 41, 42, 43)]


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("geometry", GEOMETRIES, ids=str)
@pytest.mark.parametrize("cut", range(len(CUTS)))
def test_window_attention(ctx, geometry, precision, cut):
    H, G, dim, vdim, window, pool = geometry
    n = sum(CUTS[cut])
    w = Window(ctx, precision, H, G, dim, vdim, window, pool, dim ** -0.5 * 2.0, 12.0, positions=n + 3, chunk=64, seed=cut)
    u = np.random.default_rng(cut + dim).standard_normal((n, H * dim + G * (dim + vdim)))
    want = w.want(u, CUTS[cut])
    got, at = [], 0
    for c in CUTS[cut]:
        got.append(w.feed(u[at:at + c]))
        at += c
    got = np.concatenate(got)
    assert worst(got, want) < 2e-5 if precision == "float32" else worst_row(got, want) < 0.015


@pytest.mark.parametrize("dim,vdim", [(64, 128), (128, 64), (128, 128)])
def test_long_chunk(ctx, dim, vdim):
    """Enough CTAs that every SM has one: the other cut of rows and keys over a CTA's warps."""
    w = Window(ctx, "bfloat16", 24, 6, dim, vdim, 150, 10, 2.0 / np.sqrt(dim), 12.0, positions=620, chunk=512)
    u = np.random.default_rng(dim).standard_normal((600, 24 * dim + 6 * (dim + vdim)))
    got = np.concatenate([w.feed(u[:88]), w.feed(u[88:])])
    rows = list(range(0, 600, 7)) + [599]
    q, k, v = w.split(seen_as(u, "bfloat16"))
    q, k = (seen_as(ref.head_rms_norm(x, n, w.desc.eps), "bfloat16") for x, n in ((q, w.qn), (k, w.kn)))
    want = np.concatenate([ref.window_pool_attention(q[i:i + 1], k, v, i, w.desc.scale, 12.0, 150, 10) for i in rows])
    assert worst_row(got[rows], want) < 0.015


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("softcap", [0.0, 5.0, 80.0, 200.0])
def test_softcaps(ctx, precision, softcap):
    """No cap, a tight one, one whose exponentials need a reference, one beyond the tensor-core kernels."""
    w = Window(ctx, precision, 4, 2, 64, 64, 30, 4, 0.6, softcap, positions=130, chunk=64, seed=9)
    u = np.random.default_rng(5).standard_normal((96, 4 * 64 + 2 * 128))
    got = np.concatenate([w.feed(u[:64]), *[w.feed(u[i:i + 1]) for i in range(64, 96)]])
    want = w.want(u, [64] + [1] * 32)
    assert worst(got, want) < 1e-4 if precision == "float32" else worst_row(got, want) < 0.03


def standout(w, n, query, keys, value):
    """Projections in which the query at one position matches only the keys at `keys`, whose values are `value`."""
    g = np.random.default_rng(11)
    u = g.standard_normal((n, w.H * w.dim + w.G * (w.dim + w.vdim))) * 0.1
    q, k, v = w.split(u)
    direction = np.zeros(w.dim)
    direction[: w.dim // 2] = 1.0
    k[..., : w.dim // 2] = 0.01 * g.standard_normal(k[..., : w.dim // 2].shape)  # other keys: orthogonal
    q[query] = direction
    k[keys] = direction
    v[...] = 0.01 * g.standard_normal(v.shape)
    v[keys] = value
    return u


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("how", ["prompt", "portions", "decoded"])
@pytest.mark.parametrize("window,pool,dim", [(32, 8, 64), (50, 7, 128), (16, 20, 64)])
def test_edges_of_window_and_blocks(ctx, precision, how, window, pool, dim):
    """A key just inside and just outside the window, and a block just seen and not yet seen."""
    n = 150
    i = n - 1
    e = max(b * pool + pool - 1 for b in range(n) if b * pool + pool - 1 <= i - window)  # last position of the last seen block
    block = lambda b: list(range(b * pool, (b + 1) * pool))
    b = e // pool
    cases_ = {"window_in": ([i - window + 1], True), "self": ([i], True), "far_block": (block(1), True), "block_in": (block(b), True), "block_out": (block(b + 1), False)}
    # keys that have left the window without being part of a seen block
    gap = [j for j in range(e + 1, i - window + 1)]
    if gap:
        cases_["window_out"] = ([i - window], False)
    for name, (keys, seen) in cases_.items():
        keys = [j for j in keys if j <= i]
        if name == "block_out":
            keys = [j for j in keys if j <= i - window]
            if not keys:
                continue
        w = Window(ctx, precision, 2, 1, dim, 64, window, pool, 16.0 / dim, 14.0, positions=n, chunk=160)
        u = standout(w, n, i, keys, 1.0)
        cuts = {"prompt": [n], "portions": [70, 2, 50, n - 122], "decoded": [n - 20] + [1] * 20}[how]
        at = 0
        for c in cuts:
            out = w.feed(u[at:at + c])
            at += c
        level = out[-1].mean()
        assert (level > 0.8) == seen, (name, level)
        assert level > 0.8 or level < 0.2, (name, level)


def test_a_wrong_restatement_shows(ctx):
    """Mistakes planted in the restatement (window one longer, no sink, block seen early) leave the tolerance."""
    w = Window(ctx, "float32", 4, 2, 64, 64, 24, 6, 0.125, 10.0, positions=120, chunk=120)
    u = np.random.default_rng(2).standard_normal((110, 4 * 64 + 2 * 128))
    got = w.feed(u)
    assert worst(got, w.want(u)) < 2e-5
    saved = ref.window_positions, ref.pooled_blocks, ref.sink_softmax
    wrong = {"window_positions": lambda i, s: saved[0](i, s + 1), "pooled_blocks": lambda i, s, p: saved[1](i, s - 1, p), "sink_softmax": lambda s: np.exp(s - s.max()) / np.exp(s - s.max()).sum()}
    for name, fn in wrong.items():
        try:
            setattr(ref, name, fn)
            assert worst(got, w.want(u)) > 1e-3, name
        finally:
            ref.window_positions, ref.pooled_blocks, ref.sink_softmax = saved


# ── whole models ────────────────────────────────────────────────────────────
def open_decoder(ctx, name, precision, max_chunk=64, seed=0, **kw):
    cfg = cases.ALL[name]
    t = cases.tensors(cfg, seed)
    arch = checkpoint.architecture(cfg)
    return arch.decoder(ctx, arch.parse(cfg), checkpoint.TensorFile(cases.stored(t)), precision=precision, max_chunk=max_chunk, **kw), ref.Pesedra(cfg, t)


LIMIT = {"float32": 1e-5, "bfloat16": 0.025}  # of worst_row
_reference = {}


def reference_logits(name, m, toks):
    key = (name, tuple(toks.tolist()))
    if key not in _reference:
        m.reset()
        _reference[key] = m.feed(toks)
    return _reference[key]


def run_cuts(dec, toks, cuts):
    out, at = [], 0
    for c in cuts:
        out.append(dec.feed(toks[at:at + c], at, range(c)))
        at += c
    assert at == len(toks)
    return np.concatenate(out)


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
def test_cache_is_used_again_without_clearing(ctx, precision):
    """Sequences of several lengths one after the other: what an earlier one left is never seen."""
    dec, m = open_decoder(ctx, "mixed", precision)
    for n, seed, cuts in ((140, 3, [139, 1]), (1, 4, [1]), (23, 5, [2, 21]), (90, 6, [60] + [1] * 30), (140, 3, [1] * 20 + [120])):
        toks = cases.tokens(cases.MIXED, n, seed)
        assert worst_row(run_cuts(dec, toks, cuts), reference_logits("mixed", m, toks)) < LIMIT[precision]


def test_only_wanted_rows(ctx):
    dec, m = open_decoder(ctx, "odd", "float32", max_chunk=32)
    toks = cases.tokens(cases.ODD, 90)
    want = reference_logits("odd", m, toks)
    places = [64, 3, 89, 31, 32, 3]
    assert worst(dec.feed(toks, 0, places), want[places]) < LIMIT["float32"]
    assert dec.feed(toks[:1], 0, []).shape == (0, 97)
    with pytest.raises(ValueError):
        dec.feed(toks[:4], 0, [4])
    with pytest.raises(capi.SmeltError):
        dec.feed([97, 1], 0, [0])  # an id past the vocabulary
    with pytest.raises(capi.SmeltError):
        dec.feed(toks[:2], 639, [0])  # positions past the table


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
    assert worst(dec.feed(toks[-2:-1], len(toks) - 2, [0]), logits[-1:]) < 1e-3
    clear = np.diff(np.sort(logits, 1)[:, -2:], axis=1)[:, 0] > 1e-3 * logits.std()
    np.testing.assert_array_equal(toks[1:][8:][clear[8:]], logits.argmax(1)[8:][clear[8:]])


def test_table_step_equals_graph_step(ctx):
    dec, _ = open_decoder(ctx, "mixed", "bfloat16")
    toks = cases.tokens(cases.MIXED, 40, 2)
    eager = []
    for i, t in enumerate(toks):
        dec.decode_step([t], i)
        eager.append(dec.logits(1)[0])
    np.testing.assert_array_equal(run_cuts(dec, toks, [1] * 40), np.stack(eager))


def test_snapshot_restores_the_whole_state(ctx):
    dec, _ = open_decoder(ctx, "mixed", "bfloat16")
    toks = cases.tokens(cases.MIXED, 120, 3)
    dec.feed(toks[:100], 0, [])
    snap = dec.capture_snapshot(100)
    first = run_cuts_from(dec, toks, 100)
    dec.feed(cases.tokens(cases.MIXED, 120, 4), 0, [])
    dec.restore_snapshot(snap)
    np.testing.assert_array_equal(run_cuts_from(dec, toks, 100), first)
    snap.close()


def run_cuts_from(dec, toks, start):
    return np.concatenate([dec.feed(toks[i:i + 1], i, [0]) for i in range(start, len(toks))])


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
    m = ref.Pesedra(cfg, t)
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
