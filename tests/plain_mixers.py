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


def wavelength_frequencies(rot):
    """Per-pair angular frequency when short wavelengths stay, long ones are stretched by `factor`, and those between are blended."""
    f = rot["base"] ** (-2.0 * np.arange(rot["dims"] // 2) / rot["dims"])
    sc = rot["scaling"]
    out = np.zeros_like(f)
    for i, v in enumerate(f):
        turns = sc["original"] * v / (2 * math.pi)  # of the pair over the original context
        if turns > sc["high"]:
            out[i] = v
        elif turns < sc["low"]:
            out[i] = v / sc["factor"]
        else:
            keep = (turns - sc["low"]) / (sc["high"] - sc["low"])
            out[i] = keep * v + (1 - keep) * v / sc["factor"]
    return out


def pair_frequencies(rot):
    if "high" in rot.get("scaling", {}):
        return wavelength_frequencies(rot), 1.0
    return yarn_frequencies(rot)


def rotate_pairs(x, pos, rot):
    """Interleaved pairs (2i, 2i + 1) of the first rot.dims entries of the last axis, by the position of the row (axis 0)."""
    f, mag = pair_frequencies(rot)
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


# ---- grouped-query attention under a window with kept first tokens, mixtures with identity experts -----------------------------
def rotate_halves(x, pos, dims, base):
    """Dimension i of the first `dims` is paired with i + dims / 2; rows (axis 0) at positions `pos`, heads on axis 1."""
    half = dims // 2
    a = np.asarray(pos, np.float64)[:, None] * base ** (-2.0 * np.arange(half) / dims)[None, :]
    cos, sin = np.cos(a)[:, None], np.sin(a)[:, None]
    y = np.array(x, np.float64)
    u, v = x[..., :half], x[..., half:dims]
    y[..., :half] = u * cos - v * sin
    y[..., half:dims] = v * cos + u * sin
    return y


def visible(query_pos, keys, size, keep_first):
    """[queries, keys]: key j is seen from i when j <= i and it is nearer than `size` or one of the first `keep_first`."""
    i, j = np.asarray(query_pos)[:, None], np.arange(keys)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def sink_attention(q, k, v, scale, seen, sink):
    """q: [T, H, D]; k: [S, G, D]; v: [S, G, E]; seen: [T, S]; sink: [H] logits that take weight and give no value."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, q[:, h] @ k[:, g].T * scale, -np.inf)
        m = np.maximum(s.max(axis=1), sink[h])[:, None]
        e = np.exp(s - m)
        out[:, h] = e / (e.sum(axis=1, keepdims=True) + np.exp(sink[h] - m)) @ v[:, g]
    return out


def gated_silu(x, gate, up, down):
    return linear(silu(linear(x, gate)) * linear(x, up), down)


def squared_relu(x, up, down):
    return linear(np.maximum(linear(x, up), 0.0) ** 2, down)


def choose_experts(z, correction, groups, keep, top):
    """One token's router logits -> [(expert, weight)]: softmax scores, choice by score + correction inside the best groups."""
    s = np.exp(z - z.max())
    s /= s.sum()
    choice = s + correction
    size = len(z) // groups
    best = sorted(range(groups), key=lambda g: -choice[g * size : (g + 1) * size].max())[:keep]
    allowed = [e for e in range(len(z)) if e // size in best]
    return [(e, s[e]) for e in sorted(allowed, key=lambda e: -choice[e])[:top]]


class PlainTenetar:
    """Norms on both sides of every sublayer; attention layers that may read an earlier layer's keys and values; dense or
    mixture feed-forwards."""

    def __init__(self, config, w):
        self.c = config
        self.w = {n: np.asarray(a, np.float64) for n, a in w.items()}
        self.eps = config["norm"]["eps"]

    def new_state(self):
        return {"pos": 0, "layers": [dict() for _ in self.c["layers"]]}

    def attention(self, i, x, layers, first):
        """`layers`: the states of all layers (this one's keys and values are appended to its own, if it has any)."""
        mx, p, w, T = self.c["layers"][i]["mixer"], "l%d.mix." % i, self.w, len(x)
        H, G, D, E, rot = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["rot"]
        pos = first + np.arange(T)
        q = rms_norm(linear(x, w[p + "q"]), self.eps, w[p + "q.norm"]).reshape(T, H, D)
        q = rotate_halves(q, pos, rot["dims"], rot["base"])
        src = mx.get("kv_from")
        st = layers[i if src is None else src]
        if src is None:
            k = rms_norm(linear(x, w[p + "k"]), self.eps, w[p + "k.norm"]).reshape(T, G, D)
            k = rotate_halves(k, pos, rot["dims"], rot["base"])
            v = linear(x, w[p + "v"]).reshape(T, G, E)
            st["k"] = np.concatenate([st["k"], k]) if st else k
            st["v"] = np.concatenate([st["v"], v]) if "v" in st else v
        seen = visible(pos, len(st["k"]), mx["mask"]["size"], mx["mask"]["keep_first"])
        o = sink_attention(q, st["k"], st["v"], mx["scale"], seen, w[p + "sink"])
        return linear(o.reshape(T, H * E), w[p + "o"])

    def mixture(self, p, mlp, x):
        w, r = self.w, mlp["router"]
        z = linear(x, w[p + "router"])
        y = np.zeros((len(x), x.shape[1]))
        for t in range(len(x)):
            for e, s in choose_experts(z[t], w[p + "correction"], r["groups"]["count"], r["groups"]["keep"], r["top"]):
                y[t] += s * (x[t] if e >= r["experts"] else squared_relu(x[t], w[p + "e%d.up" % e], w[p + "e%d.down" % e]))
        return y + sigmoid(linear(x, w[p + "shared.sg"])) * squared_relu(x, w[p + "shared.up"], w[p + "shared.down"])

    def feed_forward(self, i, x):
        mlp, p = self.c["layers"][i]["mlp"], "l%d.mlp." % i
        if mlp["kind"] == "moe":
            return self.mixture(p, mlp, x)
        return gated_silu(x, self.w[p + "gate"], self.w[p + "up"], self.w[p + "down"])

    def forward(self, tokens, state, trace=None):
        first, w = state["pos"], self.w
        x = w["embed"][np.asarray(tokens)] * self.c["embedding"]["scale"]
        norm = lambda name, v: rms_norm(v, self.eps, w[name])
        for i, ly in enumerate(self.c["layers"]):
            l = "l%d." % i
            x = x + norm(l + "norm1b", self.attention(i, norm(l + "norm1", x), state["layers"], first))
            if ly["mlp"] is not None:
                x = x + norm(l + "norm2b", self.feed_forward(i, norm(l + "norm2", x)))
            if trace is not None:
                trace.append(x.copy())
        state["pos"] = first + len(tokens)
        return linear(norm("final.norm", x), w["head"])


# ---- attention beside a linear recurrence, per-layer token inputs, sigmoid-scored mixtures -----------------------------------
def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def capped_attention(q, k, v, scale, first, cap):
    """Causal softmax attention of H query heads over G key/value heads; scores bounded by cap * tanh(s / cap) unless cap is None."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    late = np.arange(k.shape[0])[None, :] > (first + np.arange(T))[:, None]
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * scale
        if cap is not None:
            s = cap * np.tanh(s / cap)
        s[late] = -np.inf
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = e / e.sum(axis=1, keepdims=True) @ v[:, h // (H // G)]
    return out


def decayed_sums(q, k, v, decay, state):
    """One head: state = decay[t] * state + k[t] v[t]^T, read with q[t].  q, k: [T, n]; v: [T, e]; state: [n, e], changed in place."""
    out = np.zeros_like(v)
    for t in range(len(v)):
        state *= decay[t]
        state += np.outer(k[t], v[t])
        out[t] = q[t] @ state
    return out


def norm_in_parts(x, parts, eps):
    """Every one of `parts` equal stretches of a row divided by its own root mean square."""
    return rms_norm(x.reshape(len(x), parts, -1), eps).reshape(x.shape)


def choose_by_sigmoid(z, correction, groups, keep, top):
    """One token's router logits -> [(expert, weight)]: the groups with the largest sums of two choice scores stay."""
    s = sigmoid(z)
    choice = s + correction
    size = len(z) // groups
    rank = [np.sort(choice[g * size : (g + 1) * size])[-2:].sum() for g in range(groups)]
    best = np.argsort(-np.array(rank), kind="stable")[:keep]
    allowed = [e for e in range(len(z)) if e // size in best]
    return [(e, s[e]) for e in sorted(allowed, key=lambda e: -choice[e])[:top]]


class PlainMunisun:
    """Layers of two mixers side by side on the same input; norms (weights stored around zero) on both sides of every sublayer; a
    part of a per-token table joins after the feed-forward."""

    def __init__(self, config, w):
        self.c = config
        self.w = {n: np.asarray(a, np.float64) for n, a in w.items()}
        self.eps = config["norm"]["eps"]

    def new_state(self):
        return {"pos": 0, "layers": [dict() for _ in self.c["layers"]]}

    def norm(self, name, x):
        return rms_norm(x, self.eps, 1.0 + self.w[name])

    def attend(self, mx, q, k, v, st, first):
        st["k"] = np.concatenate([st["k"], k]) if "k" in st else k
        st["v"] = np.concatenate([st["v"], v]) if "v" in st else v
        return capped_attention(q, st["k"], st["v"], mx["scale"], first, mx.get("softcap")).reshape(len(q), -1)

    def gated_attention(self, p, mx, x, st, first):
        """Norms per head ahead of the rotation; an output gate."""
        T, H, G, D, E, w = len(x), mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], self.w
        pos = first + np.arange(T)
        q = rotate_pairs(rms_norm(linear(x, w[p + "q"]).reshape(T, H, D), self.eps, w[p + "q.norm"]), pos, mx["rot"])
        k = rotate_pairs(rms_norm(linear(x, w[p + "k"]).reshape(T, G, D), self.eps, w[p + "k.norm"]), pos, mx["rot"])
        o = self.attend(mx, q, k, linear(x, w[p + "v"]).reshape(T, G, E), st, first)
        return linear(o * sigmoid(linear(x, w[p + "g"])), w[p + "o"])

    def conv_attention(self, p, mx, x, st, first):
        """Short convolutions on the projections; norms without weights behind the rotation."""
        T, H, G, D, E, w = len(x), mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], self.w
        pos = first + np.arange(T)
        u = {}
        for n in "qkv":
            y = linear(x, w[p + n])
            u[n], st["tail." + n] = causal_conv(y, w[p + n + ".conv"], st.get("tail." + n, np.zeros((mx["conv"] - 1, y.shape[1]))))
        q = rms_norm(rotate_pairs(u["q"].reshape(T, H, D), pos, mx["rot"]), self.eps)
        k = rms_norm(rotate_pairs(u["k"].reshape(T, G, D), pos, mx["rot"]), self.eps)
        return linear(self.attend(mx, q, k, u["v"].reshape(T, G, E), st, first), w[p + "o"])

    def state_space(self, p, mx, x, st):
        T, H, E, N, G, w = len(x), mx["heads"], mx["vdim"], mx["state"], mx["groups"], self.w
        inner = H * E
        z = linear(x, w[p + "in"])
        gate, u, dt = z[:, :inner], z[:, inner : 2 * inner + 2 * G * N], z[:, 2 * inner + 2 * G * N :]
        if not st:
            st["tail"], st["S"] = np.zeros((mx["conv"] - 1, u.shape[1])), np.zeros((H, N, E))
        u, st["tail"] = causal_conv(u, w[p + "conv"], st["tail"])
        u = silu(u + w[p + "conv.b"])
        v, b, c = u[:, :inner].reshape(T, H, E), u[:, inner : inner + G * N].reshape(T, G, N), u[:, inner + G * N :].reshape(T, G, N)
        dt = softplus(dt + w[p + "dt_bias"])
        y = np.zeros((T, H, E))
        for h in range(H):
            g = h // (H // G)
            decay = np.exp(-np.exp(w[p + "A_log"][h]) * dt[:, h])
            y[:, h] = decayed_sums(c[:, g], b[:, g], v[:, h] * dt[:, h : h + 1], decay, st["S"][h]) + w[p + "D"][h] * v[:, h]
        y = norm_in_parts(y.reshape(T, inner) * silu(gate), mx["norm_groups"], self.eps) * w[p + "norm"]
        return linear(y, w[p + "o"])

    def lightning(self, p, mx, x, st):
        T, H, D, E, w = len(x), mx["heads"], mx["dim"], mx["vdim"], self.w
        q, k, v = (silu(linear(x, w[p + n])).reshape(T, H, -1) for n in "qkv")
        if not st:
            st["S"] = np.zeros((H, D, E))
        o = np.zeros((T, H, E))
        for h in range(H):
            o[:, h] = decayed_sums(q[:, h], k[:, h], v[:, h], np.full(T, mx["decay"][h]), st["S"][h])
        o = rms_norm(o.reshape(T, H * E), self.eps, w[p + "norm"]) * sigmoid(linear(x, w[p + "g"]))
        return linear(o, w[p + "o"])

    def mix(self, i, x, st, first):
        ly, p, w = self.c["layers"][i], "l%d.mix." % i, self.w
        m = ly["mixer"]
        left, right = st.setdefault("left", {}), st.setdefault("right", {})
        if ly["type"] == "parallel":
            return m["left_scale"] * self.gated_attention(p + "left.", m["left"], x, left, first) + m["right_scale"] * self.state_space(p + "right.", m["right"], x, right)
        a, b = self.conv_attention(p + "left.", m["left"], x, left, first), self.lightning(p + "right.", m["right"], x, right)
        return 0.5 * (rms_norm(a, self.eps, w[p + "left.out"]) + rms_norm(b, self.eps, w[p + "right.out"]))

    def feed_forward(self, i, x):
        mlp, p, w = self.c["layers"][i]["mlp"], "l%d.mlp." % i, self.w
        if mlp["kind"] == "dense":
            return gated_silu(x, w[p + "gate"], w[p + "up"], w[p + "down"])
        r, y = mlp["router"], np.zeros_like(x)
        z = linear(x, w[p + "router"])
        for t in range(len(x)):
            for e, s in choose_by_sigmoid(z[t], w[p + "correction"], r["groups"]["count"], r["groups"]["keep"], r["top"]):
                y[t] += s * gated_silu(x[t], w[p + "e%d.gate" % e], w[p + "e%d.up" % e], w[p + "e%d.down" % e])
        return y

    def token_side(self, i, x, tokens):
        """What the layer's part of the side table adds to the residual."""
        p, w, n = "l%d.side." % i, self.w, self.c["token_side"]["dim"]
        e = w["side.embed"][np.asarray(tokens), i * n : (i + 1) * n]
        return rms_norm(linear(gelu_tanh(linear(x, w[p + "gate"])) * e, w[p + "proj"]), self.eps, w[p + "norm"])

    def forward(self, tokens, state, trace=None):
        first, w = state["pos"], self.w
        x = w["embed"][np.asarray(tokens)] * self.c["embedding"]["scale"]
        for i, ly in enumerate(self.c["layers"]):
            l = "l%d." % i
            x = x + self.norm(l + "norm1b", self.mix(i, self.norm(l + "norm1", x), state["layers"][i], first))
            if ly["mlp"] is not None:
                x = x + self.norm(l + "norm2b", self.feed_forward(i, self.norm(l + "norm2", x)))
            x = x + self.token_side(i, x, tokens)
            if trace is not None:
                trace.append(x.copy())
        state["pos"] = first + len(tokens)
        return linear(self.norm("final.norm", x), w["head"])


# ---- delta rule with separate removal, attention with biases and a gate per head, token pairs, averages over depth ---------------
def general_delta_rule(r, k, v, w, a, state, unit_eps=1e-6):
    """One head: the state loses its part along the unit key (each key channel at its own rate a) and fades by w, both seen from the
    state before the token; then the token is added and the result read with r.  r, k, v, w, a: [T, n]; state: [n, n], changed in place."""
    out = np.zeros_like(v)
    for t in range(len(v)):
        u = unit(k[t], unit_eps)
        held = u @ state
        state *= w[t][:, None]
        state -= np.outer(a[t] * u, held)
        state += np.outer(k[t], v[t])
        out[t] = r[t] @ state
    return out


def query_temperature(pos, temp):
    """Factor on the queries at positions `pos`."""
    return 1.0 + temp["coef"] * np.log(np.floor((np.asarray(pos) + 1) / temp["every"]) + 1.0)


def masked_attention(q, k, v, scale, cap, seen):
    """Softmax over the keys in `seen` [T, S]; H query heads over G key/value heads; scores bounded unless cap is None."""
    H, G = q.shape[1], k.shape[1]
    out = np.zeros(q.shape[:2] + (v.shape[2],))
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * scale
        if cap is not None:
            s = cap * np.tanh(s / cap)
        s = np.where(seen, s, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = e / e.sum(axis=1, keepdims=True) @ v[:, h // (H // G)]
    return out


def rotate_half_pairs(x, pos, rot):
    """Dimension i of the first rot.dims is paired with i + dims / 2; frequencies and magnitude of the config's scaling."""
    f, mag = yarn_frequencies(rot)
    half = rot["dims"] // 2
    a = np.asarray(pos, np.float64)[:, None, None] * f
    cos, sin = np.cos(a) * mag, np.sin(a) * mag
    u, v = x[..., :half], x[..., half : 2 * half]
    return np.concatenate([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half :]], axis=-1)


def pair_rows(tokens, before, bigram):
    """Row of the pair table for every token; `before`: the token ahead of the first one, None at the start of a sequence."""
    rows, prev = [], before
    for t in tokens:
        rows.append(bigram["buckets"] if prev is None else (int(prev) * bigram["mul_prev"] + int(t) * bigram["mul_cur"]) % bigram["buckets"])
        prev = t
    return rows


def gated_gelu(x, gate, up, down):
    return linear(gelu_tanh(linear(x, gate)) * linear(x, up), down)


class PlainNepudra:
    """Norms (one number each) on the sublayers' inputs; behind every layer a weighted sum of the embedding and all layers' results."""

    def __init__(self, config, w):
        self.c = config
        self.w = {n: np.asarray(a, np.float64) for n, a in w.items()}
        self.eps = config["norm"]["eps"]

    def new_state(self):
        return {"pos": 0, "last": None, "layers": [dict() for _ in self.c["layers"]]}

    def norm(self, name, x):
        return rms_norm(x, self.eps) * self.w[name].reshape(())

    def general_delta(self, i, x, st):
        m, p, w, T = self.c["layers"][i]["mixer"], "l%d.mix." % i, self.w, len(x)
        H, D = m["heads"], m["dim"]
        heads = lambda z: z.reshape(T, H, D)
        r, k, v = (heads(linear(x, w[p + n])) for n in "rkv")
        decay = heads(np.exp(-np.exp(-0.5) * sigmoid(linear(np.tanh(linear(x, w[p + "w1"])), w[p + "w2"]) + w[p + "w0"])))
        a = heads(sigmoid(linear(x, w[p + "a"]) + w[p + "a.b"]))
        if not st:
            st["S"] = np.zeros((H, D, D))
        o = np.stack([general_delta_rule(r[:, h], k[:, h], v[:, h], decay[:, h], a[:, h], st["S"][h]) for h in range(H)], axis=1)
        o = rms_norm(o, self.eps).reshape(T, H * D) * w[p + "norm"]
        return linear(o * sigmoid(linear(x, w[p + "g"])), w[p + "o"])

    def attention(self, i, x, layers, first):
        """Both kinds: `layers` holds all layers' states."""
        ly = self.c["layers"][i]
        m, p, w, T = ly["mixer"], "l%d.mix." % i, self.w, len(x)
        H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        pos = first + np.arange(T)
        second = ly["type"] == "attention_2"

        def placed(z, n):
            if second:
                z = rms_norm(z, self.eps, w[p + n + ".norm"])
            return rotate_half_pairs(z, pos, m["rot"]) if "rot" in m else z

        q = placed((linear(x, w[p + "q"]) + w[p + "q.b"]).reshape(T, H, D), "q")
        if "q_temp" in m:
            q = q * query_temperature(pos, m["q_temp"])[:, None, None]
        src = m.get("kv_from")
        st = layers[i if src is None else src]
        if src is None:
            k = placed((linear(x, w[p + "k"]) + w[p + "k.b"]).reshape(T, G, D), "k")
            v = (linear(x, w[p + "v"]) + w[p + "v.b"]).reshape(T, G, E)
            st["k"] = np.concatenate([st["k"], k]) if "k" in st else k
            st["v"] = np.concatenate([st["v"], v]) if "v" in st else v
        size = m["mask"]["size"] if "mask" in m else first + T
        o = masked_attention(q, st["k"], st["v"], m["scale"], m.get("softcap"), visible(pos, len(st["k"]), size, 0))
        o = o * sigmoid(linear(x, w[p + "g"]))[:, :, None]
        y = linear(o.reshape(T, H * E), w[p + "o"])
        return y if second else y + w[p + "o.b"]

    def mix(self, i, x, layers, first):
        if self.c["layers"][i]["type"] == "general_delta":
            return self.general_delta(i, x, layers[i])
        return self.attention(i, x, layers, first)

    def feed_forward(self, i, x):
        p, w = "l%d.mlp." % i, self.w
        return gated_gelu(x, w[p + "gate"], w[p + "up"], w[p + "down"])

    def embed(self, tokens, state):
        x = self.w["embed"][np.asarray(tokens)] + self.w["bigram"][pair_rows(tokens, state["last"], self.c["embedding"]["bigram"])]
        state["last"] = tokens[-1]
        return x

    def forward(self, tokens, state, trace=None):
        first = state["pos"]
        x = self.embed(tokens, state)
        depth = [x]
        for i, ly in enumerate(self.c["layers"]):
            l = "l%d." % i
            x = x + self.mix(i, self.norm(l + "norm1", x), state["layers"], first)
            if ly["mlp"] is not None:
                x = x + self.feed_forward(i, self.norm(l + "norm2", x))
            depth.append(x)
            x = sum(c * y for c, y in zip(self.w[l + "dwa"], depth))
            if trace is not None:
                trace.append(x.copy())
        state["pos"] = first + len(tokens)
        return linear(self.norm("final.norm", x), self.w["head"])


def plain_model(config, w):
    return {"Varasun": PlainModel, "Tenetar": PlainTenetar, "Munisun": PlainMunisun, "Nepudra": PlainNepudra}[config["architecture"]](config, w)
