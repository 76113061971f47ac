"""Plain float64 restatement of the Kesedra decoder, one function per mechanism.

Slow on purpose and free of any product code: every query walks its keys one by one from the whole
history, the recurrence goes token by token, every token visits its experts one by one.  The tests
compare the CUDA path with it.

Notation: x is the residual stream [T, width], h a normed copy of it; i a query position, j a key
position; S the state of one recurrent head, [key channel, value channel].
"""
from __future__ import annotations

import json

import numpy as np

from .pesedra import read_safetensors


def linear(w, x):
    return x @ np.asarray(w, np.float64).T


# ── mechanisms ──────────────────────────────────────────────────────────────
def embed(table, tokens, scale):
    return table[tokens].astype(np.float64) * scale


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, -1, keepdims=True) + eps)


def zero_centred_norm(x, w, eps):
    """RMS norm with the weight stored around zero."""
    return unit_rms(x, eps) * (1.0 + w.astype(np.float64))


def plain_norm(x, w, eps):
    return unit_rms(x, eps) * w.astype(np.float64)


def rotate_interleaved(x, positions, base, dims):
    """x [T, ..., n]: the pairs (2i, 2i+1) of its first `dims` elements turned by p base^(-2i/dims)."""
    out = np.array(x, np.float64)
    for t, p in enumerate(positions):
        for i in range(dims // 2):
            a = float(p) * base ** (-2.0 * i / dims)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * np.cos(a) - v * np.sin(a)
            out[t, ..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def softmax(s):
    e = np.exp(s - np.max(s))
    return e / e.sum()


def window_positions(i, size):
    return range(max(0, i - size + 1), i + 1)


def latent_window_attention(q, qr, c, kr, uk, uv, first, scale, size):
    """q [n, H, dim] and rotated qr [n, H, rot] at positions first ..; latents c [T, rank] and rotated
    key parts kr [T, rot] of every position so far; uk [H, dim, rank], uv [H, vdim, rank].
    Returns [n, H, vdim]."""
    n, H, _ = q.shape
    out = np.zeros((n, H, uv.shape[1]))
    for r in range(n):
        near = list(window_positions(first + r, size))
        for h in range(H):
            k, v = c[near] @ uk[h].T, c[near] @ uv[h].T
            out[r, h] = softmax((k @ q[r, h] + kr[near] @ qr[r, h]) * scale) @ v
    return out


def token_shift(h, before):
    """The previous token's h for every token; `before` precedes the first."""
    return np.concatenate([before[None], h[:-1]])


def mixed(h, shifted, mu):
    return h + (shifted - h) * mu.astype(np.float64)


def silu(z):
    return z / (1.0 + np.exp(-z))


def decay(mix, w1, w2, w0):
    return np.exp(-np.exp(linear(w2, np.tanh(linear(w1, mix))) + w0.astype(np.float64)))


def wkv(r, k, v, w, u, state):
    """r, k, v, w [T, H, dim], u [H, dim], state [H, dim, dim].  Returns (o [T, H, dim], state)."""
    state = np.array(state, np.float64)
    out = np.zeros_like(v)
    for t in range(r.shape[0]):
        for h in range(r.shape[1]):
            now = np.outer(k[t, h], v[t, h])
            out[t, h] = (state[h] + u[h][:, None] * now).T @ r[t, h]
            state[h] = w[t, h][:, None] * state[h] + now
    return out, state


def dense_ff(h, up, up_b, down, down_b):
    return linear(down, np.maximum(linear(up, h) + up_b, 0.0) ** 2) + down_b


def route(h, router, bias, top):
    """(experts, weights), each [T, top]: the largest logits and the softmax over them alone."""
    z = linear(router, h) + bias
    chosen = np.argsort(-z, -1, kind="stable")[:, :top]
    return chosen, np.stack([softmax(z[t, chosen[t]]) for t in range(len(z))])


def expert(h, gate, up, down, limit):
    g, u = np.minimum(linear(gate, h), limit), np.clip(linear(up, h), -limit, limit)
    return linear(down, g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0))


def moe_ff(h, router, bias, top, experts, limit):
    """experts: (gate, up, down) of each."""
    chosen, weights = route(h, router, bias, top)
    return np.stack([sum(weights[t, n] * expert(h[t], *experts[e], limit) for n, e in enumerate(chosen[t])) for t in range(len(h))])


# ── model ───────────────────────────────────────────────────────────────────
class Kesedra:
    """Keeps every latent; feed() takes the next tokens of the one sequence it holds."""

    def __init__(self, config: dict, tensors: dict):
        self.c, self.w = config, tensors
        self.eps = config["norm"]["eps"]
        self.reset()

    @classmethod
    def from_folder(cls, path: str):
        with open(path + "/config.json") as f:
            return cls(json.load(f), read_safetensors(path + "/model.safetensors"))

    def reset(self):
        self.n = 0
        self.cache = {}  # layer -> (latents, rotated key parts)
        self.state = {}  # layer -> (previous h, states of the heads)

    def latent_attention(self, i, mx, h):
        W, p, T = self.w, f"l{i}.mix", len(h)
        H, d, dr, dv, rank, rot = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"], mx["rot"]
        pos = self.n + np.arange(T)
        q = linear(W[p + ".uq"], plain_norm(linear(W[p + ".dq"], h), W[p + ".dq.norm"], self.eps)).reshape(T, H, d + dr)
        if "kv_from" in mx:
            c, kr = self.cache[mx["kv_from"]]
        else:
            kv = linear(W[p + ".dkv"], h)
            c = plain_norm(kv[:, :rank], W[p + ".dkv.norm"], self.eps)
            kr = rotate_interleaved(kv[:, rank:], pos, rot["base"], rot["dims"])
            if i in self.cache:
                c, kr = (np.concatenate(a) for a in zip(self.cache[i], (c, kr)))
            self.cache[i] = (c, kr)
        a = latent_window_attention(q[..., :d], rotate_interleaved(q[..., d:], pos, rot["base"], rot["dims"]), c, kr,
                                    W[p + ".uk"].reshape(H, d, rank).astype(np.float64), W[p + ".uv"].reshape(H, dv, rank).astype(np.float64), self.n, mx["scale"], mx["mask"]["size"])
        return linear(W[p + ".o"], a.reshape(T, H * dv))

    def time_mix(self, i, mx, h):
        W, p, T, H, d = self.w, f"l{i}.mix", len(h), mx["heads"], mx["dim"]
        before, state = self.state.get(i, (np.zeros(h.shape[1]), np.zeros((H, d, d))))
        shifted = token_shift(h, before)
        mix = {s: mixed(h, shifted, W[f"{p}.mu.{s}"]) for s in "rkvgw"}
        r, k, v = (linear(W[f"{p}.{s}"], mix[s]).reshape(T, H, d) for s in "rkv")
        w = decay(mix["w"], W[p + ".w1"], W[p + ".w2"], W[p + ".w0"]).reshape(T, H, d)
        o, state = wkv(r, k, v, w, W[p + ".u"].astype(np.float64), state)
        self.state[i] = (h[-1], state)
        o = unit_rms(o, self.eps).reshape(T, H * d) * W[p + ".norm"] * silu(linear(W[p + ".g"], mix["g"]))
        return linear(W[p + ".o"], o)

    def feed_forward(self, i, mlp, h):
        W, p = self.w, f"l{i}.mlp"
        if mlp["kind"] == "dense":
            return dense_ff(h, W[p + ".up"], W[p + ".up.b"], W[p + ".down"], W[p + ".down.b"])
        experts = [tuple(W[f"{p}.e{e}.{n}"] for n in ("gate", "up", "down")) for e in range(mlp["router"]["experts"])]
        return moe_ff(h, W[p + ".router"], W[p + ".router.b"], mlp["router"]["top"], experts, mlp["expert"]["limit"])

    def feed(self, tokens, layers=None):
        """Logits [T, vocab] of the next tokens; layers: a list that receives x after every layer."""
        W, c, eps = self.w, self.c, self.eps
        tokens = np.asarray(tokens)
        x = embed(W["embed"], tokens, c["embedding"]["scale"])
        for i, L in enumerate(c["layers"]):
            mixer = self.time_mix if L["type"] == "wkv" else self.latent_attention
            x = x + zero_centred_norm(mixer(i, L["mixer"], zero_centred_norm(x, W[f"l{i}.norm1"], eps)), W[f"l{i}.norm1b"], eps)
            if L.get("mlp"):
                x = x + zero_centred_norm(self.feed_forward(i, L["mlp"], zero_centred_norm(x, W[f"l{i}.norm2"], eps)), W[f"l{i}.norm2b"], eps)
            if layers is not None:
                layers.append(x)
        self.n += len(tokens)
        return linear(W["head"], zero_centred_norm(x, W["final.norm"], eps))
