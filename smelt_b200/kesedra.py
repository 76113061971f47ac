"""Kesedra: a decoder of RWKV-style time mixing and latent window attention layers, with squared-ReLU
or mixture-of-experts feed-forwards, every sublayer between a norm before and a norm after it.

This module reads the configuration, lays the tensors out as the weights image that
``smelt_cuda_build_stack_decoder`` takes (heads, ranks and columns padded with zeros to what the
kernels want), and registers the architecture.
"""
from __future__ import annotations

from dataclasses import dataclass

import numpy as np

from . import capi, checkpoint, package

UNBOUNDED = 1 << 30  # positions: no cache grows with them


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot_base: float
    rot_dims: int
    window: int
    kv_from: int = -1


@dataclass(frozen=True)
class WkvConfig:
    heads: int
    dim: int


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    limit: float
    experts: int
    top: int


@dataclass(frozen=True)
class LayerConfig:
    mixer: object
    mlp: object  # None: no feed-forward


@dataclass(frozen=True)
class Config:
    vocab: int
    width: int
    embedding_scale: float
    eps: float
    layers: tuple


def _parse_mixer(i: int, entry: dict):
    m = entry["mixer"]
    if entry["type"] == "latent_attention":
        rot = m["rot"]
        source = m.get("kv_from")
        out = LatentConfig(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), int(m["q_rank"]), float(m["scale"]), float(rot["base"]),
                           int(rot["dims"]), int(m["mask"]["size"]), -1 if source is None else int(source))
        if min(out.heads, out.dim, out.rot_dim, out.vdim, out.kv_rank, out.q_rank, out.window) <= 0 or not 0 <= out.rot_dims <= out.rot_dim or out.rot_dims % 2 or out.rot_base <= 0:
            raise checkpoint.CheckpointError(f"layer {i}: bad sizes")
        return out
    if entry["type"] == "wkv":
        out = WkvConfig(int(m["heads"]), int(m["dim"]))
        if min(out.heads, out.dim) <= 0:
            raise checkpoint.CheckpointError(f"layer {i}: bad sizes")
        return out
    raise checkpoint.CheckpointError(f"layer {i}: unknown mixer {entry['type']!r}")


def _parse_mlp(i: int, mlp: dict | None):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        out = DenseConfig(int(mlp["ff"]))
    elif mlp["kind"] == "moe":
        out = ExpertsConfig(int(mlp["expert"]["ff"]), float(mlp["expert"]["limit"]), int(mlp["router"]["experts"]), int(mlp["router"]["top"]))
        if not 0 < out.top <= out.experts:
            raise checkpoint.CheckpointError(f"layer {i}: bad expert counts")
    else:
        raise checkpoint.CheckpointError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    if out.ff <= 0:
        raise checkpoint.CheckpointError(f"layer {i}: bad sizes")
    return out


def parse(config: dict) -> Config:
    """``config.json`` as a ``Config``; anything it asks for beyond the design is an error."""
    try:
        layers = tuple(LayerConfig(_parse_mixer(i, entry), _parse_mlp(i, entry.get("mlp"))) for i, entry in enumerate(config["layers"]))
        out = Config(int(config["vocab"]), int(config["width"]), float(config["embedding"]["scale"]), float(config["norm"]["eps"]), layers)
    except KeyError as e:
        raise checkpoint.CheckpointError(f"config.json: {e.args[0]!r} is missing") from None
    if not layers or min(out.vocab, out.width) <= 0:
        raise checkpoint.CheckpointError("config.json: bad sizes")
    for i, layer in enumerate(layers):
        m = layer.mixer
        if isinstance(m, LatentConfig) and m.kv_from >= 0:
            source = layers[m.kv_from].mixer if m.kv_from < i else None
            same = lambda a, b: (a.kv_rank, a.rot_dim, a.rot_base, a.rot_dims) == (b.kv_rank, b.rot_dim, b.rot_base, b.rot_dims)
            if not isinstance(source, LatentConfig) or source.kv_from >= 0 or not same(source, m):
                raise checkpoint.CheckpointError(f"layer {i}: layer {m.kv_from} has no cache that fits it")
    return out


def tensor_shapes(c: Config, decay_rank) -> dict:
    """name -> shape of every tensor of a model (all bfloat16).  decay_rank: layer -> inner size of its
    decay, which no configuration gives (it is the first size of the layer's ``mix.w1``)."""
    out = {"embed": (c.vocab, c.width)}
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}", layer.mixer, layer.mlp
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            out[f"{p}.{n}"] = (c.width,)
        if isinstance(m, LatentConfig):
            out[f"{p}.mix.dq"], out[f"{p}.mix.dq.norm"] = (m.q_rank, c.width), (m.q_rank,)
            out[f"{p}.mix.uq"] = (m.heads * (m.dim + m.rot_dim), m.q_rank)
            if m.kv_from < 0:
                out[f"{p}.mix.dkv"], out[f"{p}.mix.dkv.norm"] = (m.kv_rank + m.rot_dim, c.width), (m.kv_rank,)
            out[f"{p}.mix.uk"], out[f"{p}.mix.uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
            out[f"{p}.mix.o"] = (c.width, m.heads * m.vdim)
        else:
            n, rank = m.heads * m.dim, decay_rank(i)
            for s in "rkvgw":
                out[f"{p}.mix.mu.{s}"] = (c.width,)
            for s in "rkvg":
                out[f"{p}.mix.{s}"] = (n, c.width)
            out[f"{p}.mix.w1"], out[f"{p}.mix.w2"], out[f"{p}.mix.w0"] = (rank, c.width), (n, rank), (n,)
            out[f"{p}.mix.u"], out[f"{p}.mix.norm"] = (m.heads, m.dim), (n,)
            out[f"{p}.mix.o"] = (c.width, n)
        if isinstance(f, DenseConfig):
            out[f"{p}.mlp.up"], out[f"{p}.mlp.up.b"], out[f"{p}.mlp.down"], out[f"{p}.mlp.down.b"] = (f.ff, c.width), (f.ff,), (c.width, f.ff), (c.width,)
        elif isinstance(f, ExpertsConfig):
            out[f"{p}.mlp.router"], out[f"{p}.mlp.router.b"] = (f.experts, c.width), (f.experts,)
            for e in range(f.experts):
                out[f"{p}.mlp.e{e}.gate"] = out[f"{p}.mlp.e{e}.up"] = (f.ff, c.width)
                out[f"{p}.mlp.e{e}.down"] = (c.width, f.ff)
    out["final.norm"] = (c.width,)
    out["head"] = (c.vocab, c.width)
    return out


def _up(n: int, k: int) -> int:
    return -(-n // k) * k


def _value_pad(n: int) -> int:
    return next((k for k in (64, 128, 256) if n <= k), _up(n, 64))


def _pad(a: np.ndarray, *shape: int) -> np.ndarray:
    """Zeros behind each axis up to the shape."""
    return a if a.shape == shape else np.pad(a, [(0, n - s) for s, n in zip(a.shape, shape)])


def _cols(a: np.ndarray) -> np.ndarray:
    return _pad(a, a.shape[0], _up(a.shape[1], 64))


def build_image(c: Config, tensors: checkpoint.TensorFile):
    """(image bytes, StackDesc, StackLayer array, package entries)."""
    img, entries = package.WeightsImage(), []
    layers = (capi.StackLayer * len(c.layers))()
    shapes = tensor_shapes(c, lambda i: tensors.shape(f"l{i}.mix.w1")[0])
    get = lambda name: tensors.bf16(name, *shapes[name])

    def put(name: str, a: np.ndarray) -> int:
        off = img.add(a)
        entries.append((name, off, a.nbytes, a.shape))
        return off

    stream = lambda name: put(name, _pad(get(name), _up(c.width, 64)))
    for i, (layer, w) in enumerate(zip(c.layers, layers)):
        p, m, f = f"l{i}", layer.mixer, layer.mlp
        w.heads, w.dim, w.kv_from = m.heads, m.dim, -1
        w.norm1, w.norm1b = stream(f"{p}.norm1"), stream(f"{p}.norm1b")
        if isinstance(m, LatentConfig):
            w.mixer = capi.MIXER_LATENT
            w.rot_dim, w.rot_dims, w.vdim, w.kv_rank, w.q_rank, w.kv_from, w.window, w.scale = m.rot_dim, m.rot_dims, m.vdim, m.kv_rank, m.q_rank, m.kv_from, m.window, m.scale
            H, dp, rp, vp, qp, kr = m.heads, _up(m.dim, 16), _up(m.rot_dim, 16), _value_pad(m.vdim), _up(m.q_rank, 64), _up(m.kv_rank, 64)
            rows = [_pad(get(f"{p}.mix.dq"), qp, c.width)]
            if m.kv_from < 0:
                rows.append(get(f"{p}.mix.dkv"))
                w.kv_norm = put(f"{p}.mix.dkv.norm", get(f"{p}.mix.dkv.norm"))
            w.in_proj = put(f"{p}.mix.in", _cols(np.concatenate(rows)))
            w.q_norm = put(f"{p}.mix.dq.norm", _pad(get(f"{p}.mix.dq.norm"), qp))
            uq = get(f"{p}.mix.uq").reshape(H, m.dim + m.rot_dim, m.q_rank)
            w.q_proj = put(f"{p}.mix.uq", np.concatenate([_pad(uq[:, :m.dim], H, dp, qp), _pad(uq[:, m.dim:], H, rp, qp)], 1).reshape(-1, qp))
            uk, uv = get(f"{p}.mix.uk").reshape(H, m.dim, m.kv_rank), get(f"{p}.mix.uv").reshape(H, m.vdim, m.kv_rank)
            w.kv_proj = put(f"{p}.mix.ukv", np.concatenate([_pad(uk, H, dp, kr).reshape(-1, kr), _pad(uv, H, vp, kr).reshape(-1, kr)]))
            w.out_proj = put(f"{p}.mix.o", _pad(get(f"{p}.mix.o").reshape(c.width, H, m.vdim), c.width, H, vp).reshape(c.width, -1))
            w.rot_freq = put(f"{p}.mix.rot", m.rot_base ** (-2.0 * np.arange(max(1, m.rot_dims // 2)) / max(1, m.rot_dims)))
        else:
            n, group = m.heads * m.dim, _up(m.heads * m.dim, 128)
            w.mixer, w.rank = capi.MIXER_WKV, shapes[f"{p}.mix.w1"][0]
            rank = _up(w.rank, 64)
            w.in_proj = put(f"{p}.mix.in", _cols(np.concatenate([_pad(get(f"{p}.mix.{s}"), group, c.width) for s in "rkvg"] + [_pad(get(f"{p}.mix.w1"), rank, c.width)])))
            w.mu = put(f"{p}.mix.mu", np.stack([_pad(get(f"{p}.mix.mu.{s}"), _up(c.width, 64)) for s in "rkvgw"]))
            w.w2 = put(f"{p}.mix.w2", _pad(get(f"{p}.mix.w2"), n, rank))
            w.w0, w.bonus, w.head_norm = (put(f"{p}.mix.{s}", get(f"{p}.mix.{s}")) for s in ("w0", "u", "norm"))
            w.out_proj = put(f"{p}.mix.o", _cols(get(f"{p}.mix.o")))
        if f is None:
            continue
        w.norm2, w.norm2b, w.ff = stream(f"{p}.norm2"), stream(f"{p}.norm2b"), f.ff
        if isinstance(f, DenseConfig):
            w.ff_kind = capi.FF_DENSE
            w.up, w.up_bias = put(f"{p}.mlp.up", _cols(get(f"{p}.mlp.up"))), put(f"{p}.mlp.up.b", get(f"{p}.mlp.up.b"))
            w.down, w.down_bias = put(f"{p}.mlp.down", _cols(get(f"{p}.mlp.down"))), put(f"{p}.mlp.down.b", get(f"{p}.mlp.down.b"))
        else:
            w.ff_kind, w.experts, w.top, w.limit = capi.FF_EXPERTS, f.experts, f.top, f.limit
            fp, wp = _up(f.ff, 64), _up(c.width, 64)
            w.router, w.router_bias = put(f"{p}.mlp.router", _cols(get(f"{p}.mlp.router"))), put(f"{p}.mlp.router.b", get(f"{p}.mlp.router.b"))
            up, down = np.zeros((f.experts, fp, 2, wp), np.uint16), np.zeros((f.experts, c.width, fp), np.uint16)
            for e in range(f.experts):
                up[e, :f.ff, 0, :c.width], up[e, :f.ff, 1, :c.width] = get(f"{p}.mlp.e{e}.gate"), get(f"{p}.mlp.e{e}.up")
                down[e, :, :f.ff] = get(f"{p}.mlp.e{e}.down")
            w.up, w.down = put(f"{p}.mlp.gate_up", up.reshape(f.experts, 2 * fp, wp)), put(f"{p}.mlp.down", down)
    desc = capi.StackDesc(layers=len(c.layers), width=c.width, vocab=c.vocab, precision=0, eps=c.eps, embedding_scale=c.embedding_scale, embedding=put("embed", get("embed")),
                          lm_head=put("head", _cols(get("head"))), final_norm=stream("final.norm"))
    return img.tobytes(), desc, layers, entries


def decoder(ctx, c: Config, tensors: checkpoint.TensorFile, precision: str = "bfloat16", capacity: int = 0, max_chunk: int = 512) -> package.DenseDecoder:
    image, desc, layers, _ = build_image(c, tensors)
    return package.DenseDecoder(ctx, image, desc, layers, capacity=capacity or UNBOUNDED, precision=precision, max_chunk=max_chunk)


def write_package(path: str, c: Config, tensors: checkpoint.TensorFile, precision: str = "bfloat16", capacity: int = 0, max_chunk: int = 512) -> None:
    """The model as a ``.smeltpkg`` directory."""
    image, desc, layers, entries = build_image(c, tensors)
    package.write_dense_package(path, "kesedra", image, desc, layers, entries, capacity or UNBOUNDED, precision, max_chunk)


checkpoint.register("Kesedra", checkpoint.Architecture(parse, decoder, write_package))
