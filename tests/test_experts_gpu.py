"""Gated and mixture feed-forwards alone on the GPU, against the plain implementation.  The rows given are bf16 values, so
routers see the same input in both precisions."""
import numpy as np
import pytest

import layered_util as U
import plain_mixers as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]

MIXTURES = {
    "grouped": (dict(), 104),
    "one expert": (dict(experts=1, identity=0, top=1, groups=1, keep=1, ff=9, shared_ff=1), 40),
    "identity only beside one expert": (dict(experts=1, identity=7, top=3, groups=1, keep=1), 40),
    "all chosen": (dict(experts=4, identity=2, top=6, groups=2, keep=2), 64),
    "odd sizes": (dict(experts=7, identity=2, top=4, groups=3, keep=2, ff=33, shared_ff=45), 101),
    "groups of one": (dict(experts=12, identity=4, top=3, groups=16, keep=5), 72),
    "many experts": (dict(experts=100, identity=28, top=8, groups=8, keep=3, ff=40, shared_ff=136), 128),
    "more experts than threads": (dict(experts=300, identity=20, top=12, groups=1, keep=1, ff=8, shared_ff=8), 48),
    "several tiles of rows": (dict(experts=6, identity=2, top=2, groups=2, keep=1, ff=200, shared_ff=264), 136),
    "long rows": (dict(experts=5, identity=1, top=2, groups=3, keep=2, ff=700, shared_ff=96), 1032),
}


def one_layer(kw, width, seed=1, correction=0.1):
    cfg = U.tenetar_config([U.with_experts(U.attention(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2), **kw)], width=width)
    return cfg, U.tenetar_weights(cfg, seed, correction=correction)


def rows(n, width, seed=0):
    return U.bf16_round(np.random.default_rng(70 + seed).normal(size=(n, width)))


def clear_calls(m, x):
    """Rows at which no two candidates for a choice are so close that 32-bit rounding could swap them."""
    mlp, w = m.c["layers"][0]["mlp"], m.w
    r = mlp["router"]
    keep = []
    n, size = r["groups"]["keep"], len(w["l0.mlp.correction"]) // r["groups"]["count"]
    for t, z in enumerate(P.linear(x.astype(np.float64), w["l0.mlp.router"])):
        s = np.exp(z - z.max())
        c = (s / s.sum() + w["l0.mlp.correction"]).reshape(-1, size)
        order = np.argsort(-c.max(axis=1))
        g, inside = c.max(axis=1)[order], np.sort(c[order[:n]].ravel())[::-1]
        gaps = [v[i - 1] - v[i] for v, i in ((g, n), (inside, r["top"])) if i < len(v)]
        if min(gaps, default=1.0) > 2e-6:
            keep.append(t)
    assert len(keep) > 0.9 * len(x)
    return keep


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MIXTURES)
def test_mixture(gpu, name, dtype):
    kw, width = MIXTURES[name]
    cfg, w = one_layer(kw, width)
    eng, m = U.engine(gpu, cfg, w, dtype), P.plain_model(cfg, w)
    for T in (1, 2, 9, 70, 301):
        x = rows(T, width, T)
        keep = clear_calls(m, x)
        U.check(eng.probe_ffn(0, x)[keep], m.feed_forward(0, x.astype(np.float64))[keep], dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("favoured", [[3], [0, 5], [7], [6, 7], [2, 7]])
def test_crowded_and_empty_experts(gpu, favoured, dtype):
    """Corrections that send every token to the same experts (one list as long as the call, the others empty), or to identity
    experts only (no product at all)."""
    kw = dict(experts=6, identity=2, top=len(favoured), groups=1, keep=1, ff=72, shared_ff=16)
    cfg, w = one_layer(kw, 96)
    w["l0.mlp.correction"] = np.where(np.isin(np.arange(8), favoured), 4.0, -4.0).astype(np.float32)
    eng, m = U.engine(gpu, cfg, w, dtype), P.plain_model(cfg, w)
    for T in (1, 17, 130, 600):
        x = rows(T, 96, T)
        U.check(eng.probe_ffn(0, x), m.feed_forward(0, x.astype(np.float64)), dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_corrections_choose_but_do_not_weigh(gpu, dtype):
    """Large corrections of either sign: dropped groups lose even to choice scores far below zero, and the weights stay scores."""
    cfg, w = one_layer(dict(experts=9, identity=3, top=4, groups=4, keep=2, ff=40, shared_ff=24), 88)
    w["l0.mlp.correction"] = U.bf16_round(np.array([-9, -9, -8.5, -7, -8, -7.5, -2, -50, -60, -40, -70, -45.0]))
    eng, m = U.engine(gpu, cfg, w, dtype), P.plain_model(cfg, w)
    x = rows(50, 88)
    picks = {e for z in P.linear(x.astype(np.float64), m.w["l0.mlp.router"]) for e, _ in P.choose_experts(z, m.w["l0.mlp.correction"], 4, 2, 4)}
    assert picks == {6, 3, 5, 4}
    U.check(eng.probe_ffn(0, x), m.feed_forward(0, x.astype(np.float64)), dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_gate_of_the_shared_expert(gpu, dtype):
    cfg, w = one_layer(dict(), 104, 4)
    for gain in (0.0, -30.0, 30.0):
        w["l0.mlp.shared.sg"] = U.bf16_round(np.full((1, 104), gain / 104))
        eng, m = U.engine(gpu, cfg, w, dtype), P.plain_model(cfg, w)
        x = rows(20, 104) + 1.0
        x = U.bf16_round(x)
        keep = clear_calls(m, x)
        U.check(eng.probe_ffn(0, x)[keep], m.feed_forward(0, x.astype(np.float64))[keep], dtype)
        eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,width,T", [(1, 8, 1), (65, 72, 3), (128, 200, 17), (48, 1000, 65), (320, 136, 300), (7, 101, 129)])
def test_gated_silu(gpu, ff, width, T, dtype):
    cfg = U.tenetar_config([U.with_ff(U.attention(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2), ff)], width=width)
    w = U.tenetar_weights(cfg, ff)
    eng, m = U.engine(gpu, cfg, w, dtype, max_seq_len=512), P.plain_model(cfg, w)
    x = rows(T, width, ff)
    U.check(eng.probe_ffn(0, x), m.feed_forward(0, x.astype(np.float64)), dtype)
    eng.close()


GATED = {
    "grouped": (dict(), 104),
    "one expert": (dict(experts=1, top=1, groups=1, keep=1, ff=9), 40),
    "groups of one": (dict(experts=12, top=3, groups=12, keep=5), 72),
    "groups of two": (dict(experts=12, top=4, groups=6, keep=2, ff=33), 101),
    "no groups": (dict(experts=9, top=4, groups=1, keep=1, ff=40), 64),
    "all kept": (dict(experts=8, top=8, groups=4, keep=4), 64),
    "many experts": (dict(experts=128, top=8, groups=8, keep=3, ff=40), 128),
    "more experts than threads": (dict(experts=320, top=12, groups=16, keep=4, ff=8), 48),
    "several tiles of rows": (dict(experts=6, top=2, groups=2, keep=1, ff=200), 136),
    "long rows": (dict(experts=6, top=2, groups=3, keep=2, ff=700), 1032),
}


def gated_layer(kw, width, seed=1, correction=0.1):
    small = U.normed_pair(U.conv_attention(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2), U.lightning((0.9,), dim=8, vdim=8))
    cfg = U.munisun_config([U.with_gated_experts(small, **kw)], width=width)
    return cfg, U.munisun_weights(cfg, seed, correction=correction)


def clear_sigmoid_calls(m, x):
    r, w = m.c["layers"][0]["mlp"]["router"], m.w
    keep, G = [], r["groups"]["count"]
    for t, z in enumerate(P.linear(x.astype(np.float64), w["l0.mlp.router"])):
        c = (P.sigmoid(z) + w["l0.mlp.correction"]).reshape(G, -1)
        rank = np.sort(c, axis=1)[:, -2:].sum(axis=1)
        order = np.argsort(-rank)
        inside = np.sort(c[order[: r["groups"]["keep"]]].ravel())[::-1]
        gaps = [v[i - 1] - v[i] for v, i in ((rank[order], r["groups"]["keep"]), (inside, r["top"])) if i < len(v)]
        if min(gaps, default=1.0) > 2e-6:
            keep.append(t)
    assert len(keep) > 0.9 * len(x)
    return keep


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", GATED)
def test_gated_mixture(gpu, name, dtype):
    kw, width = GATED[name]
    cfg, w = gated_layer(kw, width)
    eng, m = U.engine(gpu, cfg, w, dtype), P.plain_model(cfg, w)
    for T in (1, 2, 9, 70, 301):
        x = rows(T, width, T)
        keep = clear_sigmoid_calls(m, x)
        U.check(eng.probe_ffn(0, x)[keep], m.feed_forward(0, x.astype(np.float64))[keep], dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("favoured", [[3], [0, 5], [6, 7, 2]])
def test_crowded_and_empty_gated_experts(gpu, favoured, dtype):
    cfg, w = gated_layer(dict(experts=8, top=len(favoured), groups=1, keep=1, ff=72), 96)
    w["l0.mlp.correction"] = np.where(np.isin(np.arange(8), favoured), 4.0, -4.0).astype(np.float32)
    eng, m = U.engine(gpu, cfg, w, dtype), P.plain_model(cfg, w)
    for T in (1, 17, 130, 600):
        x = rows(T, 96, T)
        U.check(eng.probe_ffn(0, x), m.feed_forward(0, x.astype(np.float64)), dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_groups_rank_by_two_and_corrections_do_not_weigh(gpu, dtype):
    """Group 0 has the single largest choice score, groups 1 and 2 the larger sums; all choice scores are negative, so a dropped expert
    that counted as zero would win."""
    cfg, w = gated_layer(dict(experts=9, top=4, groups=3, keep=2, ff=40), 88)
    w["l0.mlp.correction"] = U.bf16_round(np.array([-3, -60, -61, -14, -12, -40, -10, -17, -18.0]))
    eng, m = U.engine(gpu, cfg, w, dtype), P.plain_model(cfg, w)
    x = rows(50, 88)
    picks = {e for z in P.linear(x.astype(np.float64), m.w["l0.mlp.router"]) for e, _ in P.choose_by_sigmoid(z, m.w["l0.mlp.correction"], 3, 2, 4)}
    assert picks == {6, 4, 3, 7}
    U.check(eng.probe_ffn(0, x), m.feed_forward(0, x.astype(np.float64)), dtype)
    eng.close()
