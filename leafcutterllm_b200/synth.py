"""Synthetic models of the benchmark shapes: which tensors exist, their ggml types and GGUF dims.

Weights are N(0, 0.02) from the library's counter-based generator keyed by (seed, tensor name,
element index) and quantised in GGUF block order; norm gains are 1.0.  The same description
feeds the CUDA engine (tensors synthesised on the device or uploaded from the host generator)
and any checker that wants the identical bytes.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from typing import Iterator, Tuple

import numpy as np

from ._capi import TYPE_BF16, TYPE_F16, TYPE_F32, TYPE_Q4_0, TYPE_Q4_K, TYPE_Q6_K, TYPE_Q8_0, check, load

SIGMA = 0.02
WEIGHT_SEED = 1234
PROMPT_SEED = 4321


@dataclass
class ModelSpec:
    name: str
    num_layers: int
    hidden_size: int
    num_heads: int
    num_kv_heads: int
    intermediate_size: int
    vocab_size: int
    rope_theta: float = 10000.0
    layer_type: int = TYPE_Q4_K
    embed_type: int = TYPE_Q4_K
    head_type: int = TYPE_Q4_K
    tied_head: bool = False
    mix: str = ""        # "q4_k_m": the type mix of such a file (see mixed_type) instead of layer_type / head_type throughout
    n_experts: int = 0   # > 0: a mixture-of-experts FFN in every layer (f32 router + n_experts SwiGLU experts, top_k of them per token)
    top_k: int = 0

    @property
    def head_dim(self) -> int:
        return self.hidden_size // self.num_heads

    def mixed_type(self, layer: int, which: str) -> int:
        """The type of attn_v / ffn_down of a layer (which = "v" | "down") and of the head (layer = -1).  With mix = "q4_k_m":
        Q6_K for the head and, for attn_v and ffn_down, in the first and last eighth of the layers and every third layer
        between; Q4_K elsewhere -- the placement the usual quantisation tool gives its "Q4_K_M" files."""
        if self.mix != "q4_k_m":
            return self.head_type if layer < 0 else self.layer_type
        if layer < 0:
            return TYPE_Q6_K
        n = self.num_layers
        more = layer < n // 8 or layer >= 7 * n // 8 or (layer - n // 8) % 3 == 2
        return TYPE_Q6_K if more else TYPE_Q4_K

    def tensors(self) -> Iterator[Tuple[str, int, Tuple[int, ...], str]]:
        """(gguf name, ggml type, dims fastest-first, 'normal' | 'ones')"""
        H, F, V = self.hidden_size, self.intermediate_size, self.vocab_size
        nq, nkv = self.num_heads * self.head_dim, self.num_kv_heads * self.head_dim
        yield "token_embd.weight", self.embed_type, (H, V), "normal"
        yield "output_norm.weight", TYPE_F32, (H,), "ones"
        if not self.tied_head:
            yield "output.weight", self.mixed_type(-1, "head"), (H, V), "normal"
        for l in range(self.num_layers):
            p = f"blk.{l}."
            yield p + "attn_norm.weight", TYPE_F32, (H,), "ones"
            yield p + "attn_q.weight", self.layer_type, (H, nq), "normal"
            yield p + "attn_k.weight", self.layer_type, (H, nkv), "normal"
            yield p + "attn_v.weight", self.mixed_type(l, "v"), (H, nkv), "normal"
            yield p + "attn_output.weight", self.layer_type, (nq, H), "normal"
            yield p + "ffn_norm.weight", TYPE_F32, (H,), "ones"
            if self.n_experts > 0:
                yield p + "ffn_gate_inp.weight", TYPE_F32, (H, self.n_experts), "normal"
                for e in range(self.n_experts):
                    q = f"{p}expert.{e}."
                    yield q + "ffn_gate.weight", self.layer_type, (H, F), "normal"
                    yield q + "ffn_up.weight", self.layer_type, (H, F), "normal"
                    yield q + "ffn_down.weight", self.layer_type, (F, H), "normal"
                continue
            yield p + "ffn_gate.weight", self.layer_type, (H, F), "normal"
            yield p + "ffn_up.weight", self.layer_type, (H, F), "normal"
            yield p + "ffn_down.weight", self.mixed_type(l, "down"), (F, H), "normal"

    def with_layers(self, n: int) -> "ModelSpec":
        import dataclasses
        return dataclasses.replace(self, num_layers=n, name=f"{self.name}-L{n}")


# TinyLlama-1.1B shape: Q4_0 layers, Q8_0 embedding and head.
TINY = ModelSpec("tinyllama-1.1b-shape-q4_0", 22, 2048, 32, 4, 5632, 32000, 10000.0, TYPE_Q4_0, TYPE_Q8_0, TYPE_Q8_0)
# Llama-2-7B shape, Q4_K throughout.
LLAMA7B = ModelSpec("llama2-7b-shape-q4_k", 32, 4096, 32, 32, 11008, 32000, 10000.0, TYPE_Q4_K, TYPE_Q4_K, TYPE_Q4_K)
# Llama-2-7B shape with the type mix of a "Q4_K_M" file: Q6_K head, Q6_K attn_v and ffn_down in about half of the layers.
LLAMA7B_Q4KM = ModelSpec("llama2-7b-shape-q4_k_m", 32, 4096, 32, 32, 11008, 32000, 10000.0, TYPE_Q4_K, TYPE_Q4_K, TYPE_Q4_K, mix="q4_k_m")
# Mixtral-8x7B shape: 8 experts of FFN 14336, two per token, 32 q / 8 kv heads, Q4_K (router f32).
MIXTRAL = ModelSpec("mixtral-8x7b-shape-q4_k", 32, 4096, 32, 8, 14336, 32000, 10000.0, TYPE_Q4_K, TYPE_Q4_K, TYPE_Q4_K, n_experts=8, top_k=2)
# Llama-3-70B shape, Q4_K.
LLAMA70B = ModelSpec("llama3-70b-shape-q4_k", 80, 8192, 64, 8, 28672, 128256, 500000.0, TYPE_Q4_K, TYPE_Q4_K, TYPE_Q4_K)


@dataclass
class LayeredSpec:
    """A checkpoint-directory model: the parsed config.json with the ranks that only the tensors' shapes give (Varasun:
    decay_rank, gate_rank), for random weights."""
    name: str
    config: dict
    decay_rank: int = 0
    gate_rank: int = 0

    @property
    def vocab_size(self) -> int:
        return self.config["vocab"]

    def tensors(self) -> Iterator[Tuple[str, int, Tuple[int, ...], str]]:
        """(checkpoint name, ggml type, dims fastest-first, 'normal' | 'ones')"""
        c = self.config
        W = c["width"]
        def mat(name, rows, cols):
            return name, TYPE_BF16, (cols, rows), "normal"
        def vec(name, n, kind="ones"):
            return name, TYPE_BF16, (n,), kind
        munisun, nepudra = c["architecture"] == "Munisun", c["architecture"] == "Nepudra"
        gain = "zeros" if munisun else "ones"  # Munisun's layer norms are stored around zero
        yield mat("embed", c["vocab"], W)
        if nepudra:
            yield mat("bigram", c["embedding"]["bigram"]["buckets"] + 1, W)
        if munisun:
            yield mat("side.embed", c["vocab"], len(c["layers"]) * c["token_side"]["dim"])
        for i, ly in enumerate(c["layers"]):
            m, p = ly["mixer"], f"l{i}.mix."
            H, D, E = (0, 0, 0) if munisun else (m["heads"], m["dim"], m.get("vdim", m["dim"]))
            both = ("", "b") if c["architecture"] in ("Tenetar", "Munisun") else ("",)  # norms on inputs and outputs, or on one of them
            wide = 1 if nepudra else W
            for end in both:
                yield vec(f"l{i}.norm1{end}", wide, gain)
            if nepudra:
                yield vec(f"l{i}.dwa", i + 2)
            if ly["type"] == "general_delta":
                for t in "rkvga":
                    yield mat(p + t, H * D, W)
                yield vec(p + "a.b", H * D, "normal")
                yield mat(p + "w1", self.decay_rank, W)
                yield mat(p + "w2", H * D, self.decay_rank)
                yield vec(p + "w0", H * D, "normal")
                yield vec(p + "norm", H * D)
                yield mat(p + "o", W, H * D)
            elif nepudra:
                G, second = m["kv_heads"], ly["type"] == "attention_2"
                for t, n in (("q", H * D), ("k", G * D), ("v", G * E)):
                    if t == "q" or "kv_from" not in m:
                        yield mat(p + t, n, W)
                        yield vec(p + t + ".b", n, "normal")
                        if second and t != "v":
                            yield vec(p + t + ".norm", D)
                yield mat(p + "g", H, W)
                yield mat(p + "o", W, H * E)
                if not second:
                    yield vec(p + "o.b", W, "normal")
            elif munisun:
                a, r, left, right = m["left"], m["right"], p + "left.", p + "right."
                nq, nk, nv, inner = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"], r["heads"] * r["vdim"]
                for t, n in (("q", nq), ("k", nk), ("v", nv)):
                    yield mat(left + t, n, W)
                    if "conv" in a:
                        yield mat(left + t + ".conv", n, a["conv"])
                yield mat(left + "o", W, a["heads"] * a["vdim"])
                if ly["type"] == "parallel":
                    yield vec(left + "q.norm", a["dim"])
                    yield vec(left + "k.norm", a["dim"])
                    yield mat(left + "g", a["heads"] * a["vdim"], W)
                    channels = inner + 2 * r["groups"] * r["state"]
                    yield mat(right + "in", inner + channels + r["heads"], W)
                    yield mat(right + "conv", channels, r["conv"])
                    yield vec(right + "conv.b", channels, "normal")
                    for t in ("dt_bias", "A_log", "D"):
                        yield vec(right + t, r["heads"], "normal")
                else:
                    for t, n in (("q", r["heads"] * r["dim"]), ("k", r["heads"] * r["dim"]), ("v", inner), ("g", inner)):
                        yield mat(right + t, n, W)
                    yield vec(left + "out", W)
                    yield vec(right + "out", W)
                yield vec(right + "norm", inner)
                yield mat(right + "o", W, inner)
                n = c["token_side"]["dim"]
                yield mat(f"l{i}.side.gate", n, W)
                yield mat(f"l{i}.side.proj", W, n)
                yield vec(f"l{i}.side.norm", W)
            elif ly["type"] == "attention":
                G = m["kv_heads"]
                yield mat(p + "q", H * D, W)
                yield vec(p + "q.norm", H * D)
                if "kv_from" not in m:
                    yield mat(p + "k", G * D, W)
                    yield vec(p + "k.norm", G * D)
                    yield mat(p + "v", G * E, W)
                yield vec(p + "sink", H)
                yield mat(p + "o", W, H * E)
            elif ly["type"] == "channel_delta":
                nk = m["kv_heads"] * D
                for t, n in (("q", nk), ("k", nk), ("v", H * E)):
                    yield mat(p + t, n, W)
                    yield mat(p + t + ".conv", n, m["conv"])
                yield mat(p + "b", H, W)
                yield vec(p + "A_log", H, "normal")
                yield vec(p + "norm", E)
                yield mat(p + "a1", self.decay_rank, W)
                yield mat(p + "a2", H * D, self.decay_rank)
                yield vec(p + "dt_bias", H * D, "normal")
                yield mat(p + "g1", self.gate_rank, W)
                yield mat(p + "g2", H * E, self.gate_rank)
                yield mat(p + "o", W, H * E)
            else:
                C_, R, Q = m["kv_rank"], m["rot_dim"], m["q_rank"]
                yield mat(p + "dq", Q, W)
                yield vec(p + "dq.norm", Q)
                yield mat(p + "uq", H * (D + R), Q)
                yield mat(p + "dkv", C_ + R, W)
                yield vec(p + "dkv.norm", C_)
                yield mat(p + "uk", H * D, C_)
                yield mat(p + "uv", H * E, C_)
                yield mat(p + "o", W, H * E)
            mlp, p = ly["mlp"], f"l{i}.mlp."
            if mlp is None:
                continue
            for end in both:
                yield vec(f"l{i}.norm2{end}", wide, gain)
            if mlp["kind"] == "moe":
                r, F, SF = mlp["router"], mlp["expert"]["ff"], mlp.get("shared", {}).get("ff", 0)
                n = r["experts"] + r.get("identity", 0)
                yield mat(p + "router", n, W)
                yield vec(p + "correction", n, "zeros")  # random routers are balanced as they are
                for e in range(r["experts"]):
                    if munisun:
                        yield mat(f"{p}e{e}.gate", F, W)
                    yield mat(f"{p}e{e}.up", F, W)
                    yield mat(f"{p}e{e}.down", W, F)
                if not SF:
                    continue
                yield mat(p + "shared.up", SF, W)
                yield mat(p + "shared.down", W, SF)
                yield mat(p + "shared.sg", 1, W)
                continue
            F = mlp["ff"]
            if c["architecture"] != "Varasun":
                yield mat(p + "gate", F, W)
            yield mat(p + "up", F, W)
            yield mat(p + "down", W, F)
        yield vec("final.norm", 1 if nepudra else W, gain)
        yield mat("head", c["vocab"], W)


def layered_spec(name: str, width: int, pattern: str, ff: int, vocab: int, heads: int, head_dim: int = 128, q_rank: int = 1536, kv_rank: int = 512,
                 rot_dim: int = 64, low_rank: int = 128) -> LayeredSpec:
    """pattern: one letter per layer, d = gated delta rule, a = latent attention, each with a feed-forward of `ff`."""
    delta = {"heads": heads, "kv_heads": heads, "dim": head_dim, "vdim": head_dim, "conv": 4}
    latent = {"heads": heads, "dim": head_dim, "rot_dim": rot_dim, "vdim": head_dim, "kv_rank": kv_rank, "q_rank": q_rank,
              "scale": (head_dim + rot_dim) ** -0.5,
              "rot": {"dims": rot_dim, "base": 10000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    layers = [{"type": "channel_delta" if ch == "d" else "latent_attention", "mixer": dict(delta if ch == "d" else latent),
               "mlp": {"kind": "dense", "ff": ff}} for ch in pattern]
    config = {"architecture": "Varasun", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "logit_softcap": 30.0, "layers": layers}
    return LayeredSpec(name, config, low_rank, low_rank)


def tenetar_spec(name: str, width: int, pattern: str, ff: int, vocab: int, heads: int, kv_heads: int, experts: int, identity: int, top: int, groups: int,
                 keep: int, expert_ff: int, shared_ff: int, head_dim: int = 128, window: int = 1024, keep_first: int = 16) -> LayeredSpec:
    """pattern: one letter per layer, d = dense feed-forward, m = mixture, s = mixture, keys and values of the last layer that has
    its own."""
    layers, own = [], 0
    for i, ch in enumerate(pattern):
        mixer = {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5,
                 "rot": {"dims": head_dim, "base": 10000.0}, "mask": {"size": window, "keep_first": keep_first}}
        if ch == "s":
            mixer["kv_from"] = own
        else:
            own = i
        moe = {"kind": "moe", "expert": {"ff": expert_ff}, "shared": {"ff": shared_ff},
               "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}}}
        layers.append({"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ch == "d" else moe})
    return LayeredSpec(name, {"architecture": "Tenetar", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5}, "layers": layers})


def munisun_spec(name: str, width: int, pattern: str, ff: int, vocab: int, heads: int, kv_heads: int, experts: int, top: int, groups: int, keep: int, expert_ff: int,
                 head_dim: int = 128, space_heads: int = 0, space_dim: int = 64, space_state: int = 128, space_groups: int = 8, side: int = 256) -> LayeredSpec:
    """pattern: two letters per layer: s = attention beside a state space, l = attention beside lightning attention; then d = dense
    feed-forward, m = mixture, n = none."""
    layers = []
    space_heads = space_heads or 2 * width // space_dim
    for kind, mlp in zip(pattern[::2], pattern[1::2]):
        left = {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5, "rot": {"dims": head_dim, "base": 500000.0}}
        if kind == "s":
            left["rot"]["scaling"] = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}
            mixer = {"left": dict(left, softcap=50.0), "left_scale": 1.0, "right_scale": 1.0,
                     "right": {"heads": space_heads, "vdim": space_dim, "state": space_state, "groups": space_groups, "conv": 4, "norm_groups": space_groups}}
        else:
            mixer = {"left": dict(left, conv=4), "right": {"heads": heads, "dim": head_dim, "vdim": head_dim, "decay": [1.0 - 2.0 ** (-3.0 - 8.0 * h / heads) for h in range(heads)]}}
        moe = {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}
        layers.append({"type": "parallel" if kind == "s" else "parallel_2", "mixer": mixer, "mlp": {"d": {"kind": "dense", "ff": ff}, "m": moe, "n": None}[mlp]})
    return LayeredSpec(name, {"architecture": "Munisun", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5}, "token_side": {"dim": side}, "layers": layers})


def nepudra_spec(name: str, width: int, pattern: str, ff: int, vocab: int, heads: int, kv_heads: int, head_dim: int = 128, state_dim: int = 64, rank: int = 64,
                 window: int = 1024, buckets: int = 32003) -> LayeredSpec:
    """pattern: one letter per layer: g = delta rule with separate removal, w = unrotated attention over everything, s = the same on the
    last w's keys and values, n = windowed attention with norms per head; each with a gated feed-forward of `ff`."""
    layers, own = [], 0
    for i, ch in enumerate(pattern):
        mixer = {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5}
        if ch == "g":
            mixer = {"heads": width // state_dim, "dim": state_dim}
        elif ch == "n":
            mixer.update(mask={"size": window}, rot={"dims": head_dim, "base": 500000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}})
        else:
            mixer.update(softcap=50.0, q_temp={"coef": 0.1, "every": 4096})
            if ch == "s":
                mixer["kv_from"] = own
            else:
                own = i
        layers.append({"type": {"g": "general_delta", "n": "attention_2"}.get(ch, "attention"), "mixer": mixer, "mlp": {"kind": "dense", "ff": ff}})
    config = {"architecture": "Nepudra", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "embedding": {"bigram": {"buckets": buckets, "mul_prev": 40503, "mul_cur": 1}}, "layers": layers}
    return LayeredSpec(name, config, rank)


def build_layered_engine(spec: LayeredSpec, seed: int = WEIGHT_SEED, **engine_kwargs):
    """An `Engine` holding the synthetic model, every tensor synthesised on the device."""
    from .engine import Engine
    eng = Engine.from_config(spec.config, **engine_kwargs)
    for name, typ, dims, kind in spec.tensors():
        if kind in ("ones", "zeros"):
            eng.set_tensor(name, TYPE_F32, dims, np.full(int(np.prod(dims)), float(kind == "ones"), np.float32))
        else:
            eng.synth_tensor(name, typ, dims, seed, SIGMA)
    eng.finalize()
    return eng


def host_tensor(typ: int, seed: int, name: str, n_elems: int, sigma: float = SIGMA) -> np.ndarray:
    """Raw block bytes of a synthetic tensor from the host generator (same bytes as the device one)."""
    lib = load()
    out = np.empty(lib.lc_tensor_bytes(typ, n_elems), np.uint8)
    check(lib.lc_synth_tensor_host(typ, seed, name.encode(), sigma, n_elems, out.ctypes.data_as(C.c_void_p)))
    return out


def tensor_bytes(spec: ModelSpec, name: str, typ: int, dims, kind: str, seed: int = WEIGHT_SEED) -> np.ndarray:
    n = int(np.prod(dims))
    if kind == "ones":
        return np.ones(n, np.float32).view(np.uint8)
    return host_tensor(typ, seed, name, n)


def prompt_tokens(n: int, vocab: int, seq_index: int = 0, seed: int = PROMPT_SEED) -> np.ndarray:
    out = np.empty(n, np.int64)
    check(load().lc_synth_tokens(seed + seq_index, n, vocab, out.ctypes.data_as(C.c_void_p)))
    return out


def build_engine(spec: ModelSpec, max_seq_len: int, seed: int = WEIGHT_SEED, on_device: bool = True, **engine_kwargs):
    """An `Engine` holding the synthetic model.  on_device=True synthesises every tensor with a CUDA
    kernel (no host copy); False runs the host generator and uploads."""
    from .engine import Engine
    eng = Engine(spec.hidden_size, spec.num_layers, spec.num_heads, spec.num_kv_heads, spec.intermediate_size,
                 spec.vocab_size, max_seq_len=max_seq_len, rope_theta=spec.rope_theta, n_experts=spec.n_experts, top_k=spec.top_k,
                 **engine_kwargs)
    for name, typ, dims, kind in spec.tensors():
        if kind == "ones" or not on_device:
            eng.set_tensor(name, typ, dims, tensor_bytes(spec, name, typ, dims, kind, seed))
        else:
            eng.synth_tensor(name, typ, dims, seed, SIGMA)
    eng.finalize()
    return eng
