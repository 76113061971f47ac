"""Plain float64 restatement of the Pesedra decoder, one function per mechanism.

Slow on purpose and free of any product code: every query walks its keys one by one, every block
mean is taken from the whole history.  The tests compare the CUDA path with it.

Notation: x is the residual stream [T, width], h a normed copy of it; i a query position, j a key
position; b a pooled block of P positions [bP, bP + P); S the window.
"""
from __future__ import annotations

import json
import struct

import numpy as np


# ── model folder ────────────────────────────────────────────────────────────
def read_safetensors(path: str) -> dict:
    """name -> array; bfloat16 widened to float32 (exact)."""
    with open(path, "rb") as f:
        raw = f.read()
    n = struct.unpack("<Q", raw[:8])[0]
    out = {}
    for name, t in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        data = raw[8 + n + lo:8 + n + hi]
        if t["dtype"] == "BF16":
            a = (np.frombuffer(data, "<u2").astype(np.uint32) << 16).view(np.float32)
        else:
            a = np.frombuffer(data, {"F32": "<f4", "I32": "<i4", "F16": "<f2"}[t["dtype"]])
        out[name] = a.reshape(t["shape"])
    return out


# ── mechanisms ──────────────────────────────────────────────────────────────
def embed(table, pos_table, tokens, positions, scale):
    return table[tokens].astype(np.float64) * scale + pos_table[positions].astype(np.float64)


def scalar_rms_norm(x, gain, eps):
    """RMS norm whose weight is one number."""
    return x / np.sqrt(np.mean(x * x, -1, keepdims=True) + eps) * float(gain)


def head_rms_norm(x, weight, eps):
    """Per head: x [..., heads, dim], one weight of size dim for all heads."""
    return x / np.sqrt(np.mean(x * x, -1, keepdims=True) + eps) * weight.astype(np.float64)


def softcapped(scores, cap):
    return cap * np.tanh(scores / cap)


def sink_softmax(scores):
    """exp(s) over one more than the sum of the exponentials."""
    if len(scores) == 0:
        return scores
    m = max(0.0, float(np.max(scores)))
    e = np.exp(scores - m)
    return e / (np.exp(-m) + e.sum())


def window_positions(i, size):
    """The positions a query at i sees one by one."""
    return range(max(0, i - size + 1), i + 1)


def pooled_blocks(i, size, pool):
    """The blocks a query at i sees: those that end at least `size` positions before it."""
    return [b for b in range(i // pool + 1) if b * pool + pool - 1 <= i - size]


def block_mean(rows, b, pool):
    return np.mean(rows[b * pool:(b + 1) * pool], axis=0)


def window_pool_attention(q, k, v, first, scale, cap, size, pool):
    """q [n, H, dim] at positions first ..; k [T, G, dim], v [T, G, vdim] of every position so far.
    Returns [n, H, vdim]."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((n, H, v.shape[2]))
    for r in range(n):
        i = first + r
        near, far = list(window_positions(i, size)), pooled_blocks(i, size, pool)
        for g in range(G):
            keys = [k[j, g] for j in near] + [block_mean(k[:, g], b, pool) for b in far]
            vals = [v[j, g] for j in near] + [block_mean(v[:, g], b, pool) for b in far]
            keys, vals = np.stack(keys), np.stack(vals)
            for h in range(g * (H // G), (g + 1) * (H // G)):
                out[r, h] = sink_softmax(softcapped(keys @ q[r, h] * scale, cap)) @ vals
    return out


def softplus(z):
    return np.log1p(np.exp(-abs(z))) + max(float(z), 0.0)


def xielu(z, p, q):
    rising, falling = softplus(float(p)), 0.5 + softplus(float(q))
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, rising * z * z, falling * (np.expm1(neg) - neg)) + z / 2


def dense_ff(h, up, down, act):
    return xielu(h @ up.T.astype(np.float64), *act) @ down.T.astype(np.float64)


def loop_entry(x, x0, w):
    """Before the first layer of a pass: a projection of [x; embedding output]."""
    return np.concatenate([x, x0], -1) @ w.T.astype(np.float64)


def layer_runs(config):
    """(layer, begins a pass) in the order of execution."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(l, False) for l in range(n)]
    body = [(l, l == loop["start"]) for l in range(loop["start"], loop["stop"])]
    return [(l, False) for l in range(loop["start"])] + body * loop["times"] + [(l, False) for l in range(loop["stop"], n)]


# ── model ───────────────────────────────────────────────────────────────────
class Pesedra:
    """Keeps every key and value; feed() takes the next tokens of the one sequence it holds."""

    def __init__(self, config: dict, tensors: dict):
        self.c, self.w = config, tensors
        self.runs = layer_runs(config)
        self.reset()

    @classmethod
    def from_folder(cls, path: str):
        with open(path + "/config.json") as f:
            return cls(json.load(f), read_safetensors(path + "/model.safetensors"))

    def reset(self):
        self.n = 0
        self.keys = [None] * len(self.runs)
        self.values = [None] * len(self.runs)

    def attention(self, run, name, mx, h):
        W, eps = self.w, self.c["norm"]["eps"]
        H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        T = h.shape[0]
        q = head_rms_norm((h @ W[name + ".q"].T.astype(np.float64)).reshape(T, H, d), W[name + ".q.norm"], eps)
        k = head_rms_norm((h @ W[name + ".k"].T.astype(np.float64)).reshape(T, G, d), W[name + ".k.norm"], eps)
        v = (h @ W[name + ".v"].T.astype(np.float64)).reshape(T, G, dv)
        self.keys[run] = k if self.keys[run] is None else np.concatenate([self.keys[run], k])
        self.values[run] = v if self.values[run] is None else np.concatenate([self.values[run], v])
        a = window_pool_attention(q, self.keys[run], self.values[run], self.n, mx["scale"], mx["softcap"], mx["mask"]["size"], mx["mask"]["pool"])
        return a.reshape(T, H * dv) @ W[name + ".o"].T.astype(np.float64)

    def feed(self, tokens, layers=None):
        """Logits [T, vocab] of the next tokens; layers: a list that receives x after every layer run."""
        W, c = self.w, self.c
        tokens = np.asarray(tokens)
        x = embed(W["embed"], W["pos"], tokens, self.n + np.arange(len(tokens)), c["embedding"]["scale"])
        x0 = x
        for run, (l, begins) in enumerate(self.runs):
            if begins:
                x = loop_entry(x, x0, W["loop.in"])
            L = c["layers"][l]
            h = scalar_rms_norm(x, W[f"l{l}.norm1"], c["norm"]["eps"])
            y = self.attention(run, f"l{l}.mix", L["mixer"], h)
            if L.get("mlp"):
                y = y + dense_ff(h, W[f"l{l}.mlp.up"], W[f"l{l}.mlp.down"], W[f"l{l}.mlp.act"])
            x = x + y
            if layers is not None:
                layers.append(x)
        self.n += len(tokens)
        return scalar_rms_norm(x, W["final.norm"], c["norm"]["eps"]) @ W["head"].T.astype(np.float64)
