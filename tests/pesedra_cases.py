"""Small Pesedra configurations and seeded weights for the tests."""
import numpy as np

from smelt_b200 import checkpoint, pesedra


def layer(heads, kv_heads, dim, vdim, size, pool, ff, scale=None, softcap=15.0):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5, "softcap": softcap,
                      "mask": {"size": size, "pool": pool}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, loop=None, max_positions=640, scale=3.0, eps=1e-5):
    c = {"architecture": "Pesedra", "embedding": {"scale": scale}, "layers": layers, "max_positions": max_positions, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# layers of unequal sizes, one without a feed-forward, an inner loop of two layers run three times
MIXED = config(width=96, vocab=131, loop=(1, 3, 3), layers=[
    layer(4, 2, 32, 48, size=24, pool=5, ff=160), layer(6, 1, 64, 32, size=40, pool=8, ff=0, softcap=9.0), layer(3, 3, 40, 64, size=17, pool=17, ff=72, scale=0.3),
    layer(8, 4, 16, 16, size=64, pool=3, ff=96)])
# a width that is no multiple of 8, many query heads on one key head, no loop, a pool longer than the window
ODD = config(width=70, vocab=97, layers=[layer(18, 1, 24, 20, size=6, pool=11, ff=50, softcap=40.0), layer(2, 2, 128, 72, size=30, pool=4, ff=33, softcap=90.0)], scale=0.7, eps=1e-3)
# wide heads, the whole stack looped, a window of one token
WIDE = config(width=128, vocab=260, loop=(0, 2, 2), layers=[layer(4, 2, 256, 200, size=50, pool=10, ff=256), layer(2, 1, 300, 128, size=1, pool=2, ff=64)])
ALL = {"mixed": MIXED, "odd": ODD, "wide": WIDE}


def tensors(cfg: dict, seed: int = 0) -> dict:
    """name -> float32 array, exactly representable in bfloat16."""
    g = np.random.Generator(np.random.Philox(key=[seed, 77]))
    out = {}
    for name, shape in pesedra.tensor_shapes(pesedra.parse(cfg)).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm", "norm1"):
            a = 1.0 + 0.3 * g.standard_normal(shape)
        elif leaf == "act":
            a = g.uniform(-1.0, 1.0, shape)
        elif name in ("embed", "pos"):
            a = g.standard_normal(shape)
        else:
            a = g.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = round_bf16(np.asarray(a, np.float32))
    return out


def round_bf16(a) -> np.ndarray:
    a = np.asarray(a, np.float32)
    return checkpoint.bf16_to_f32(checkpoint.f32_to_bf16(a)).reshape(a.shape)


def stored(t: dict) -> dict:
    """The tensors as ``checkpoint`` reads and writes them."""
    return {k: ("BF16", checkpoint.f32_to_bf16(v).reshape(v.shape)) for k, v in t.items()}


def tokens(cfg: dict, n: int, seed: int = 1) -> np.ndarray:
    return np.random.Generator(np.random.Philox(key=[seed, 78])).integers(0, cfg["vocab"], n).astype(np.int32)
