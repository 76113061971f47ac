"""Small Kesedra configurations and seeded weights for the tests."""
import numpy as np

from pesedra_cases import round_bf16, stored, tokens  # noqa: F401  (shared by every design's cases)
from smelt_b200 import kesedra

FEATURES = 3  # stream elements that no sublayer changes: the routers read them, so that no choice of experts is a close one


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, size, mlp, kv_from=None, base=1000.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5,
         "mask": {"size": size}, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def wkv(heads, dim, mlp):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, scale=4.0, eps=1e-5):
    return {"architecture": "Kesedra", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# layers of unequal sizes in another order; one cache read by two later layers, one of them with a longer window than its owner's; a layer without a feed-forward
MIXED = config(width=96, vocab=131, layers=[
    wkv(3, 32, moe(6, 2, 40)), latent(4, 32, 16, 48, 40, 56, 24, dense(160)), latent(2, 24, 16, 32, 40, 72, 37, moe(9, 3, 24, limit=0.4), kv_from=1, scale=0.3),
    wkv(5, 16, None), latent(6, 16, 8, 16, 64, 32, 9, dense(72)), latent(3, 40, 16, 64, 40, 48, 11, dense(48), kv_from=1)])
# a width that is no multiple of 8, odd heads and sizes, one token chosen by one expert, a window of one token, long key parts
ODD = config(width=70, vocab=97, scale=0.9, eps=1e-3, layers=[
    latent(17, 20, 6, 18, 33, 27, 1, moe(3, 1, 17)), wkv(2, 33, dense(50)), latent(1, 70, 34, 100, 130, 90, 45, None), wkv(1, 72, moe(35, 2, 9, limit=3.0)),
    latent(5, 12, 6, 10, 33, 20, 30, dense(33), kv_from=0)])
# wide heads and ranks, all experts chosen, a layer that is more than its width
WIDE = config(width=192, vocab=260, layers=[latent(2, 256, 64, 300, 200, 128, 50, moe(4, 4, 130)), wkv(2, 128, dense(256)), latent(8, 64, 32, 128, 520, 100, 70, dense(64)),
                                            wkv(1, 200, moe(8, 2, 64, limit=0.7))])
ALL = {"mixed": MIXED, "odd": ODD, "wide": WIDE}
# seeds whose first tokens are well conditioned (at position 0 a head's output is (r . u k) v over its own size: a product near zero magnifies every rounding)
SEED = {"mixed": 0, "odd": 0, "wide": 1}
DECAY_RANK = {"mixed": 24, "odd": 7, "wide": 80}


def named(cfg, table):
    return next(table[n] for n, c in ALL.items() if c is cfg)


def router(g, experts: int, top: int):
    """(weights of the features, bias): of several draws the one whose choices are the clearest for all signs and sizes of the features."""
    signs = np.array([[1 if b >> j & 1 else -1 for j in range(FEATURES)] for b in range(1 << FEATURES)], np.float64)
    best = None
    for _ in range(1500):
        w, b = round_bf16(g.standard_normal((experts, FEATURES))), round_bf16(0.1 * g.standard_normal(experts))
        z = np.stack([f * signs @ w.T.astype(np.float64) + b for f in (0.3, 0.5, 0.8, 1.2, 2.0, 4.0)])  # [size, signs, experts]
        order = np.argsort(-z, -1)
        z = np.take_along_axis(z, order, -1)
        gap = float(np.min(z[..., top - 1] - z[..., top])) if top < experts else 1.0
        if (np.sort(order[..., :top], -1) != np.sort(order[:1, :, :top], -1)).any():
            gap = 0.0  # a choice changes with the features' size
        if best is None or gap > best[0]:
            best = (gap, w, b)
        if top == experts:
            break
    return best[1:]


def tensors(cfg: dict) -> dict:
    """name -> float32 array, exactly representable in bfloat16."""
    g = np.random.Generator(np.random.Philox(key=[named(cfg, SEED), 79]))
    out, c = {}, kesedra.parse(cfg)
    routers = {f"l{i}.mlp.router": router(g, layer.mlp.experts, layer.mlp.top) for i, layer in enumerate(c.layers) if isinstance(layer.mlp, kesedra.ExpertsConfig)}
    for name, shape in kesedra.tensor_shapes(c, lambda i: named(cfg, DECAY_RANK)).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            a = 0.3 * g.standard_normal(shape)  # stored around zero
            if leaf in ("norm1b", "norm2b"):
                a[:FEATURES] = -1.0  # nothing is ever added to these elements of the stream
            if leaf == "norm2":
                a[:FEATURES] = 0.0
        elif leaf == "norm":
            a = 1.0 + 0.3 * g.standard_normal(shape)
        elif ".mu." in name:
            a = g.uniform(0.0, 1.0, shape)
        elif leaf == "w0":
            a = g.uniform(-4.0, 0.5, shape)
        elif leaf == "u":
            a = g.standard_normal(shape)
        elif name.removesuffix(".b") in routers and leaf == "b":
            a = routers[name.removesuffix(".b")][1]
        elif leaf == "b":
            a = 0.5 * g.standard_normal(shape)
        elif name == "embed":
            a = g.standard_normal(shape)
            a[:, :FEATURES] = 3.0 * g.choice([-1.0, 1.0], (shape[0], FEATURES))
        elif leaf == "router":
            a = 0.02 * g.standard_normal(shape) / np.sqrt(shape[1])
            a[:, :FEATURES] = routers[name][0]
        else:
            a = g.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = round_bf16(np.asarray(a, np.float32))
    return out


def close_calls(cfg: dict, t: dict, m, toks, margin: float) -> float:
    """The share of (token, expert layer) pairs of the restatement whose last chosen and first unchosen logits are less than `margin` apart."""
    from oracle import kesedra as ref

    gaps, kept = [], ref.route

    def spy(h, router, bias, top):
        z = np.sort(ref.linear(router, h) + bias, -1)[:, ::-1]
        if top < z.shape[1]:
            gaps.append(z[:, top - 1] - z[:, top])
        return kept(h, router, bias, top)
    ref.route = spy
    try:
        m.reset()
        m.feed(toks)
    finally:
        ref.route = kept
    return float(np.mean(np.concatenate(gaps) < margin)) if gaps else 0.0
