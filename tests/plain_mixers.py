"""A plain, slow implementation of the checkpoint-directory model designs, one function per mechanism, in float64 numpy.

It is the yardstick of the GPU tests: written from the equations, token by token where the mechanism is a recurrence, and
sharing no code with the product.  Notation: rows are tokens, a linear map W of shape [out, in] is applied as x @ W.T.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def linear(x, w):
    return x @ np.asarray(w, np.float64).T


def rms_norm(x, eps, w=None):
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if w is None else y * w


def unit(x, eps=1e-6):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + eps)


def causal_conv(x, w, tail):
    """y[t] = sum_j w[:, j] x[t - (taps - 1) + j] per channel; `tail` holds the taps - 1 inputs before x.  Returns (y, new tail)."""
    taps = w.shape[1]
    full = np.concatenate([tail, x], axis=0)
    y = np.zeros_like(x)
    for j in range(taps):
        y += full[j : j + len(x)] * w[:, j]
    return y, full[len(full) - (taps - 1) :]


def delta_rule(q, k, v, g, beta, state):
    """Per head: decay the key rows of the state, write the correction towards v, read with q.
    q, k, g: [T, dim]; v: [T, vdim]; beta: [T]; state: [dim, vdim] (changed in place)."""
    out = np.zeros_like(v)
    for t in range(len(v)):
        state *= g[t][:, None]
        u = beta[t] * (v[t] - state.T @ k[t])
        state += np.outer(k[t], u)
        out[t] = state.T @ q[t]
    return out


def yarn_frequencies(rot):
    """(per-pair angular frequency, factor on cos and sin) of a rotation config."""
    dims, base = rot["dims"], rot["base"]
    i = np.arange(dims // 2)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    def dim_of(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(dim_of(sc["fast"])), 0)
    hi = min(math.ceil(dim_of(sc["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_pairs(x, pos, rot):
    """Interleaved pairs (2i, 2i + 1) of the first rot.dims entries of the last axis, by the position of the row (axis 0)."""
    f, mag = yarn_frequencies(rot)
    a = np.asarray(pos, np.float64)[:, None] * f[None, :]
    cos, sin = np.cos(a) * mag, np.sin(a) * mag
    while cos.ndim < x.ndim:
        cos, sin = cos[:, None], sin[:, None]
    y = np.array(x, np.float64)
    d = rot["dims"]
    u, v = x[..., 0:d:2], x[..., 1:d:2]
    y[..., 0:d:2] = u * cos - v * sin
    y[..., 1:d:2] = v * cos + u * sin
    return y


def causal_softmax_attention(q, k, v, scale, first):
    """q: [T, H, D] at positions first .. first + T - 1; k: [S, H, D], v: [S, H, E] at positions 0 .. S - 1."""
    s = np.einsum("thd,shd->hts", q, k) * scale
    visible = np.arange(k.shape[0])[None, :] <= (first + np.arange(q.shape[0]))[:, None]
    s = np.where(visible[None], s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    p /= p.sum(axis=-1, keepdims=True)
    return np.einsum("hts,she->the", p, v)


class PlainModel:
    """config: the parsed config.json; w: name -> array (float)."""

    def __init__(self, config, w):
        self.c = config
        self.w = {n: np.asarray(a, np.float64) for n, a in w.items()}
        self.eps = config["norm"]["eps"]

    def new_state(self):
        return {"pos": 0, "layers": [dict() for _ in self.c["layers"]]}

    def channel_delta(self, p, mx, x, st):
        T, H, KH, D, E = len(x), mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        w = self.w
        if not st:
            st["tail"] = {n: np.zeros((mx["conv"] - 1, w[p + n].shape[0])) for n in "qkv"}
            st["S"] = np.zeros((H, D, E))
        parts = {}
        for n in "qkv":
            y, st["tail"][n] = causal_conv(linear(x, w[p + n]), w[p + n + ".conv"], st["tail"][n])
            parts[n] = silu(y)
        q = unit(parts["q"].reshape(T, KH, D)) * D ** -0.5
        k = unit(parts["k"].reshape(T, KH, D))
        v = parts["v"].reshape(T, H, E)
        beta = sigmoid(linear(x, w[p + "b"]))
        a = linear(linear(x, w[p + "a1"]), w[p + "a2"]) + w[p + "dt_bias"]
        g = np.exp(-np.exp(w[p + "A_log"])[None, :, None] * softplus(a).reshape(T, H, D))
        o = np.zeros((T, H, E))
        for h in range(H):
            kh = h // (H // KH)
            o[:, h] = delta_rule(q[:, kh], k[:, kh], v[:, h], g[:, h], beta[:, h], st["S"][h])
        o = rms_norm(o, self.eps, w[p + "norm"])
        gate = sigmoid(linear(linear(x, w[p + "g1"]), w[p + "g2"])).reshape(T, H, E)
        return linear((o * gate).reshape(T, H * E), w[p + "o"])

    def latent_attention(self, p, mx, x, st, first):
        T, H, D, R, E, C = len(x), mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
        w = self.w
        if not st:
            st["c"], st["kr"] = np.zeros((0, C)), np.zeros((0, R))
        pos = first + np.arange(T)
        cq = rms_norm(linear(x, w[p + "dq"]), self.eps, w[p + "dq.norm"])
        q = linear(cq, w[p + "uq"]).reshape(T, H, D + R)
        q = np.concatenate([q[..., :D], rotate_pairs(q[..., D:], pos, mx["rot"])], axis=-1)
        z = linear(x, w[p + "dkv"])
        st["c"] = np.concatenate([st["c"], rms_norm(z[:, :C], self.eps, w[p + "dkv.norm"])])
        st["kr"] = np.concatenate([st["kr"], rotate_pairs(z[:, C:], pos, mx["rot"])])
        S = len(st["c"])
        k = linear(st["c"], w[p + "uk"]).reshape(S, H, D)
        k = np.concatenate([k, np.broadcast_to(st["kr"][:, None, :], (S, H, R))], axis=-1)
        v = linear(st["c"], w[p + "uv"]).reshape(S, H, E)
        o = causal_softmax_attention(q, k, v, mx["scale"], first)
        return linear(o.reshape(T, H * E), w[p + "o"])

    def feed_forward(self, p, x):
        return linear(np.maximum(linear(x, self.w[p + "up"]), 0.0) ** 2, self.w[p + "down"])

    def mix(self, i, x, st, first):
        ly = self.c["layers"][i]
        p = "l%d.mix." % i
        if ly["type"] == "channel_delta":
            return self.channel_delta(p, ly["mixer"], x, st)
        return self.latent_attention(p, ly["mixer"], x, st, first)

    def forward(self, tokens, state, trace=None):
        """Logits of every given token; `state` (new_state()) carries on from earlier calls."""
        first = state["pos"]
        x = self.w["embed"][np.asarray(tokens)]
        for i, ly in enumerate(self.c["layers"]):
            x = x + rms_norm(self.mix(i, x, state["layers"][i], first), self.eps, self.w["l%d.norm1" % i])
            if ly["mlp"] is not None:
                x = x + rms_norm(self.feed_forward("l%d.mlp." % i, x), self.eps, self.w["l%d.norm2" % i])
            if trace is not None:
                trace.append(x.copy())
        state["pos"] = first + len(tokens)
        z = linear(rms_norm(x, self.eps, self.w["final.norm"]), self.w["head"]) * self.c["logit_scale"]
        cap = self.c["logit_softcap"]
        return cap * np.tanh(z / cap)
