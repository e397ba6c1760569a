"""Small random checkpoint-directory models for the tests: configs, bf16 weights, checkpoint files, engines."""
import json
import os
import struct

import numpy as np


def bf16_round(a):
    """The nearest bf16 values (ties to even), as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) & np.uint32(0xFFFF0000)).view(np.float32)


def bf16_bytes(a):
    return (bf16_round(a).view(np.uint32) >> np.uint32(16)).astype(np.uint16)


def delta(heads=3, kv_heads=1, dim=24, vdim=20, conv=4):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": None}


def latent(heads=5, dim=20, rot_dim=12, vdim=18, kv_rank=28, q_rank=36, scale=0.2, base=10000.0, scaling=(3.0, 64, 8.0, 1.0)):
    rot = {"dims": rot_dim, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                  "scale": scale, "rot": rot}, "mlp": None}


def with_ff(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def config(layers, width=104, vocab=131, eps=1e-5, logit_scale=0.7, softcap=12.0):
    return {"architecture": "Varasun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale, "logit_softcap": softcap,
            "layers": layers}


def attention(heads=6, kv_heads=3, dim=20, vdim=12, rot_dims=8, base=10000.0, scale=0.3, window=37, keep_first=5, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot_dims, "base": base},
         "mask": {"size": window, "keep_first": keep_first}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None}


def with_experts(layer, experts=10, identity=2, top=3, groups=3, keep=2, ff=24, shared_ff=20):
    return dict(layer, mlp={"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared_ff},
                            "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}}})


def tenetar_config(layers, width=104, vocab=131, eps=1e-5, embed_scale=3.0):
    return {"architecture": "Tenetar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "layers": layers}


def tenetar_weights(cfg, seed=0, fixed_choice=False, correction=0.1):
    """Random weights, already rounded to bf16.  fixed_choice: corrections far larger than any score, so that the rounding of
    bf16 activations cannot change which experts are chosen (their weights still follow the token)."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    w = {}

    def mat(name, n, k, gain=1.0):
        w[name] = rng.normal(0, gain / np.sqrt(k), (n, k))

    def gain(name, n):
        w[name] = rng.normal(1, 0.2, n)

    w["embed"] = rng.normal(0, 0.4, (cfg["vocab"], W))
    for i, ly in enumerate(cfg["layers"]):
        m, l, p = ly["mixer"], "l%d." % i, "l%d.mix." % i
        H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b"):
            gain(l + n, W)
        mat(p + "q", H * D, W)
        gain(p + "q.norm", H * D)
        if m.get("kv_from") is None:
            mat(p + "k", G * D, W)
            gain(p + "k.norm", G * D)
            mat(p + "v", G * E, W)
        w[p + "sink"] = rng.normal(1.0, 1.0, H)
        mat(p + "o", W, H * E)
        mlp, p = ly["mlp"], l + "mlp."
        if mlp is None:
            continue
        for n in ("norm2", "norm2b"):
            gain(l + n, W)
        if mlp["kind"] == "dense":
            mat(p + "gate", mlp["ff"], W)
            mat(p + "up", mlp["ff"], W)
            mat(p + "down", W, mlp["ff"])
            continue
        r, F, SF = mlp["router"], mlp["expert"]["ff"], mlp["shared"]["ff"]
        n = r["experts"] + r.get("identity", 0)
        mat(p + "router", n, W, 1.5)
        w[p + "correction"] = rng.permutation(n) * 2.0 - n if fixed_choice else rng.normal(-correction, correction, n)
        for e in range(r["experts"]):
            mat(p + "e%d.up" % e, F, W, 2.0)
            mat(p + "e%d.down" % e, W, F, 2.0)
        mat(p + "shared.up", SF, W)
        mat(p + "shared.down", W, SF)
        mat(p + "shared.sg", 1, W)
    gain("final.norm", W)
    mat("head", cfg["vocab"], W, 2.0)
    return {n: bf16_round(a) for n, a in w.items()}


def tenetar_mixed():
    """Windows of several sizes, shared caches (also under a wider window than their owner's), every kind of feed-forward."""
    return tenetar_config([with_ff(attention(), 40), with_experts(attention(heads=4, kv_heads=1, dim=16, vdim=24, rot_dims=16, window=18, keep_first=0)),
                           with_experts(attention(heads=8, kv_heads=1, dim=16, vdim=24, rot_dims=16, window=50, keep_first=21, kv_from=1), experts=5, identity=3, top=4, groups=4, keep=3, ff=31),
                           attention(window=1000, keep_first=0, kv_from=0), with_ff(attention(window=9, keep_first=2, kv_from=0), 17)])


def weights(cfg, seed=0, decay_rank=5, gate_rank=7, spread=1.0):
    """Random weights, already rounded to bf16.  Products keep about unit size; decays range from slow to fast."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    w = {}

    def mat(name, n, k, gain=1.0):
        w[name] = rng.normal(0, gain * spread / np.sqrt(k), (n, k))

    def gain(name, n):
        w[name] = rng.normal(1, 0.2, n)

    w["embed"] = rng.normal(0, 1, (cfg["vocab"], W))
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], "l%d.mix." % i
        H, D, E = m["heads"], m["dim"], m["vdim"]
        gain("l%d.norm1" % i, W)
        if ly["type"] == "channel_delta":
            for t, n in (("q", m["kv_heads"] * D), ("k", m["kv_heads"] * D), ("v", H * E)):
                mat(p + t, n, W)
                w[p + t + ".conv"] = rng.normal(0, 0.6, (n, m["conv"]))
            mat(p + "b", H, W)
            w[p + "A_log"] = rng.uniform(-3, 1.5, H)
            gain(p + "norm", E)
            mat(p + "a1", decay_rank, W)
            mat(p + "a2", H * D, decay_rank, 2.0)
            w[p + "dt_bias"] = rng.uniform(-4, 2, H * D)
            mat(p + "g1", gate_rank, W)
            mat(p + "g2", H * E, gate_rank)
            mat(p + "o", W, H * E)
        else:
            C, R, Q = m["kv_rank"], m["rot_dim"], m["q_rank"]
            mat(p + "dq", Q, W)
            gain(p + "dq.norm", Q)
            mat(p + "uq", H * (D + R), Q, 2.0)
            mat(p + "dkv", C + R, W)
            gain(p + "dkv.norm", C)
            mat(p + "uk", H * D, C)
            mat(p + "uv", H * E, C)
            mat(p + "o", W, H * E)
        if ly["mlp"]:
            gain("l%d.norm2" % i, W)
            mat("l%d.mlp.up" % i, ly["mlp"]["ff"], W)
            mat("l%d.mlp.down" % i, W, ly["mlp"]["ff"])
    gain("final.norm", W)
    mat("head", cfg["vocab"], W, 2.0)
    return {n: bf16_round(a) for n, a in w.items()}


def write_checkpoint(folder, cfg, w):
    head, blob, at = {}, [], 0
    for n in sorted(w):
        b = bf16_bytes(w[n]).tobytes()
        head[n] = {"dtype": "BF16", "shape": list(w[n].shape), "data_offsets": [at, at + len(b)]}
        blob.append(b)
        at += len(b)
    text = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blob))
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)


def engine(lc, cfg, w, dtype="float32", **kw):
    from leafcutterllm_b200 import Engine
    eng = Engine.from_config(cfg, dtype=dtype, **kw)
    for n, a in w.items():
        eng.set_tensor(n, lc.TYPE_BF16, tuple(reversed(a.shape)), bf16_bytes(a))
    eng.finalize()
    return eng


def tokens(n, vocab, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, vocab, n).tolist()


def rel_rms(got, want):
    """Largest row error: rms of the difference over the rms of all expected values."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    d = np.sqrt(np.mean((got - want) ** 2, axis=-1))
    return float(d.max() / np.sqrt(np.mean(want ** 2)))


# Bounds on the error of the worst row and of all rows together: f32 rounding, and the rounding of bf16 activations.
WORST_ROW = {"float32": 3e-5, "bfloat16": 6e-2}
ALL_ROWS = {"float32": 1e-5, "bfloat16": 2e-2}


def check(got, want, dtype, slack=1):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    worst = rel_rms(got, want)
    total = float(np.sqrt(np.mean((got - want) ** 2) / np.mean(want ** 2)))
    assert worst < slack * WORST_ROW[dtype] and total < slack * ALL_ROWS[dtype], (worst, total)
