"""Pesedra: a looped decoder of parallel layers with attention over a window and pooled blocks.

Every layer adds its mixer and its feed-forward, both reading one RMS norm whose weight is a single
number, to an fp32 residual stream.  Queries and keys are normed per head and not rotated;
positions enter through a learned table.  A range of layers runs several times with the same
weights, each pass entered through a projection of [x; embedding output].

This module reads the configuration, lays the tensors out as the weights image that
``smelt_cuda_build_dense_decoder`` takes, and registers the architecture.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import numpy as np

from . import capi, checkpoint, package


@dataclass(frozen=True)
class LayerConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    pool: int
    scale: float
    softcap: float
    ff: int  # 0: no feed-forward

    @property
    def qkv(self) -> int:
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim)


@dataclass(frozen=True)
class Config:
    vocab: int
    width: int
    max_positions: int
    embedding_scale: float
    eps: float
    layers: tuple
    loop: tuple = (0, 0, 0)  # start, stop, times

    def runs(self) -> list[int]:
        """The layer of every layer run, in the order of execution."""
        start, stop, times = self.loop
        n = len(self.layers)
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))


def parse(config: dict) -> Config:
    """``config.json`` as a ``Config``; anything it asks for beyond the design is an error."""
    try:
        layers = []
        for i, entry in enumerate(config["layers"]):
            if entry["type"] != "attention":
                raise checkpoint.CheckpointError(f"layer {i}: unknown mixer {entry['type']!r}")
            m, mlp = entry["mixer"], entry.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise checkpoint.CheckpointError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["mask"]["size"]), int(m["mask"]["pool"]),
                                      float(m["scale"]), float(m["softcap"]), int(mlp["ff"]) if mlp is not None else 0))
        loop = config.get("loop")
        out = Config(int(config["vocab"]), int(config["width"]), int(config["max_positions"]), float(config["embedding"]["scale"]), float(config["norm"]["eps"]),
                     tuple(layers), (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else (0, 0, 0))
    except KeyError as e:
        raise checkpoint.CheckpointError(f"config.json: {e.args[0]!r} is missing") from None
    for i, c in enumerate(out.layers):
        if min(c.heads, c.kv_heads, c.dim, c.vdim, c.window, c.pool) <= 0 or c.heads % c.kv_heads or c.ff < 0:
            raise checkpoint.CheckpointError(f"layer {i}: bad sizes")
    if not out.layers or min(out.vocab, out.width, out.max_positions) <= 0 or not 0 <= out.loop[0] <= out.loop[1] <= len(out.layers) or out.loop[2] < 0:
        raise checkpoint.CheckpointError("config.json: bad sizes or loop")
    return out


def tensor_shapes(c: Config) -> dict:
    """name -> shape of every tensor of a model (all bfloat16)."""
    out = {"embed": (c.vocab, c.width), "pos": (c.max_positions, c.width)}
    if c.loop[1] > c.loop[0]:
        out["loop.in"] = (c.width, 2 * c.width)
    for i, m in enumerate(c.layers):
        p = f"l{i}"
        out[f"{p}.norm1"] = ()
        out[f"{p}.mix.q"] = (m.heads * m.dim, c.width)
        out[f"{p}.mix.k"] = (m.kv_heads * m.dim, c.width)
        out[f"{p}.mix.v"] = (m.kv_heads * m.vdim, c.width)
        out[f"{p}.mix.q.norm"] = out[f"{p}.mix.k.norm"] = (m.dim,)
        out[f"{p}.mix.o"] = (c.width, m.heads * m.vdim)
        if m.ff:
            out[f"{p}.mlp.up"] = (m.ff, c.width)
            out[f"{p}.mlp.down"] = (c.width, m.ff)
            out[f"{p}.mlp.act"] = (2,)
    out["final.norm"] = ()
    out["head"] = (c.vocab, c.width)
    return out


def _pad_cols(a: np.ndarray) -> np.ndarray:
    pad = -a.shape[1] % 64
    return np.pad(a, ((0, 0), (0, pad))) if pad else a


def _softplus(v: float) -> float:
    return max(v, 0.0) + math.log1p(math.exp(-abs(v)))


def build_image(c: Config, tensors: checkpoint.TensorFile):
    """(image bytes, DenseDesc, DenseLayer array): a layer's input projections as one matrix
    [q; k; v; up], its output projections as one matrix [o | down]."""
    img = package.WeightsImage()
    layers = (capi.DenseLayer * len(c.layers))()
    shapes = tensor_shapes(c)
    get = lambda name: tensors.bf16(name, *shapes[name])
    for i, m in enumerate(c.layers):
        p, w = f"l{i}", layers[i]
        w.heads, w.kv_heads, w.dim, w.vdim, w.window, w.pool, w.ff = m.heads, m.kv_heads, m.dim, m.vdim, m.window, m.pool, m.ff
        w.scale, w.softcap, w.norm_gain = m.scale, m.softcap, float(tensors.f32(f"{p}.norm1"))
        rows, cols = [get(f"{p}.mix.{n}") for n in "qkv"], [get(f"{p}.mix.o")]
        if m.ff:
            rows.append(get(f"{p}.mlp.up"))
            cols.append(get(f"{p}.mlp.down"))
            rising, falling = (float(v) for v in tensors.f32(f"{p}.mlp.act", 2))
            w.act_rising, w.act_falling = _softplus(rising), 0.5 + _softplus(falling)
        w.in_proj = img.add(_pad_cols(np.concatenate(rows)))
        w.out_proj = img.add(_pad_cols(np.concatenate(cols, 1)))
        w.q_norm, w.k_norm = img.add(get(f"{p}.mix.q.norm")), img.add(get(f"{p}.mix.k.norm"))
    desc = capi.DenseDesc(layers=len(c.layers), width=c.width, vocab=c.vocab, precision=0, max_positions=c.max_positions, loop_start=c.loop[0], loop_stop=c.loop[1],
                          loop_times=c.loop[2], eps=c.eps, embedding_scale=c.embedding_scale, final_gain=float(tensors.f32("final.norm")),
                          embedding=img.add(get("embed")), positions=img.add(get("pos")), lm_head=img.add(_pad_cols(get("head"))))
    if "loop.in" in shapes:
        w = get("loop.in")
        desc.loop_in = img.add(np.concatenate([_pad_cols(w[:, :c.width]), _pad_cols(w[:, c.width:])], 1))
    return img.tobytes(), desc, layers


def decoder(ctx, c: Config, tensors: checkpoint.TensorFile, precision: str = "bfloat16", capacity: int = 0, max_chunk: int = 512) -> package.DenseDecoder:
    image, desc, layers = build_image(c, tensors)
    return package.DenseDecoder(ctx, image, desc, layers, capacity=min(capacity or c.max_positions, c.max_positions), precision=precision, max_chunk=max_chunk)


def write_package(path: str, c: Config, tensors: checkpoint.TensorFile, precision: str = "bfloat16", capacity: int = 0, max_chunk: int = 512) -> None:
    """The model as a ``.smeltpkg`` directory."""
    image, desc, layers = build_image(c, tensors)
    pad = lambda n: -(-n // 64) * 64
    entries = [("embed", desc.embedding, c.vocab, c.width), ("pos", desc.positions, c.max_positions, c.width), ("head", desc.lm_head, c.vocab, pad(c.width))]
    if c.loop[1] > c.loop[0]:
        entries.append(("loop.in", desc.loop_in, c.width, 2 * pad(c.width)))
    for i, (m, w) in enumerate(zip(c.layers, layers)):
        entries += [(f"l{i}.in", w.in_proj, m.qkv + m.ff, pad(c.width)), (f"l{i}.out", w.out_proj, c.width, pad(m.heads * m.vdim + m.ff)),
                    (f"l{i}.q.norm", w.q_norm, 1, m.dim), (f"l{i}.k.norm", w.k_norm, 1, m.dim)]
    package.write_dense_package(path, "pesedra", image, desc, layers, [(n, off, rows * cols * 2, (rows, cols)) for n, off, rows, cols in entries],
                                min(capacity or c.max_positions, c.max_positions), precision, max_chunk)


checkpoint.register("Pesedra", checkpoint.Architecture(parse, decoder, write_package))
