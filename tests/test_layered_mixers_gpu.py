"""Every mechanism of the checkpoint-directory layers alone, on the GPU, against the plain implementation."""
import numpy as np
import pytest

import layered_util as U
import plain_mixers as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]

DELTAS = {
    "shared keys": (U.delta(heads=3, kv_heads=1, dim=24, vdim=20, conv=4), 104, 5, 7),
    "no convolution": (U.delta(heads=2, kv_heads=2, dim=16, vdim=8, conv=1), 40, 3, 9),
    "two taps, odd values": (U.delta(heads=4, kv_heads=2, dim=12, vdim=9, conv=2), 72, 8, 8),
    "long convolution": (U.delta(heads=2, kv_heads=1, dim=40, vdim=33, conv=6), 64, 11, 1),
    "large heads": (U.delta(heads=2, kv_heads=2, dim=128, vdim=128, conv=4), 256, 32, 16),
    "larger than a warp row": (U.delta(heads=1, kv_heads=1, dim=160, vdim=192, conv=3), 128, 16, 24),
}
LATENTS = {
    "uneven sizes": (U.latent(), 104),
    "no scaling": (U.latent(heads=2, dim=8, rot_dim=16, vdim=24, kv_rank=17, q_rank=9, scaling=None), 72),
    "many heads": (U.latent(heads=37, dim=16, rot_dim=8, vdim=16, kv_rank=40, q_rank=48), 128),
    "large": (U.latent(heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=96, scale=0.072), 256),
    "middle": (U.latent(heads=18, dim=64, rot_dim=32, vdim=48, kv_rank=200, q_rank=64, scale=0.1), 128),
    "wide values": (U.latent(heads=2, dim=32, rot_dim=16, vdim=136, kv_rank=136, q_rank=32), 64),
}


def one_layer(layer, width, ra=5, rg=7, seed=1):
    cfg = U.config([layer], width=width)
    return cfg, U.weights(cfg, seed, ra, rg)


def rows(n, width, seed=0):
    return U.bf16_round(np.random.default_rng(50 + seed).normal(size=(n, width)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", DELTAS)
def test_delta_layer(gpu, name, dtype):
    layer, width, ra, rg = DELTAS[name]
    cfg, w = one_layer(layer, width, ra, rg)
    eng, m = U.engine(gpu, cfg, w, dtype, max_seq_len=128), P.PlainModel(cfg, w)
    x, st = rows(77, width), {}
    for lo, hi in ((0, 40), (40, 42), (42, 43), (43, 77)):
        want = m.channel_delta("l0.mix.", layer["mixer"], x[lo:hi].astype(np.float64), st)
        U.check(eng.probe_attention(0, x[lo:hi]), want, dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", LATENTS)
def test_latent_layer(gpu, name, dtype):
    layer, width = LATENTS[name]
    cfg, w = one_layer(layer, width)
    eng, m = U.engine(gpu, cfg, w, dtype, max_seq_len=256), P.PlainModel(cfg, w)
    x, st, at = rows(201, width), {}, 0
    for n in (70, 15, 1, 16, 64, 2, 33):  # token by token up to 15 tokens, tiles from 16 on
        want = m.latent_attention("l0.mix.", layer["mixer"], x[at : at + n].astype(np.float64), st, at)
        U.check(eng.probe_attention(0, x[at : at + n]), want, dtype)
        at += n
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,width", [(40, 104), (200, 72), (1, 8), (513, 256)])
def test_squared_relu(gpu, ff, width, dtype):
    cfg, w = one_layer(U.with_ff(U.delta(), ff), width)
    eng, m = U.engine(gpu, cfg, w, dtype), P.PlainModel(cfg, w)
    x = rows(19, width)
    U.check(eng.probe_ffn(0, x), m.feed_forward("l0.mlp.", x.astype(np.float64)), dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_convolution_reaches_exactly_taps_tokens_back(gpu, dtype):
    """An impulse on one input row: outputs of the layer change from that row on, and the convolution's part of the change
    ends taps rows later (seen with decays so fast that the state forgets at once)."""
    layer = U.delta(heads=1, kv_heads=1, dim=8, vdim=8, conv=3)
    cfg, w = one_layer(layer, 32)
    w["l0.mix.dt_bias"] = np.full_like(w["l0.mix.dt_bias"], 60.0)
    w["l0.mix.A_log"] = np.full_like(w["l0.mix.A_log"], 3.0)
    eng = U.engine(gpu, cfg, w, dtype)
    x = rows(24, 32)
    base = eng.probe_attention(0, x)
    y = x.copy()
    y[9] = 0
    eng.kv_clear()
    changed = np.abs(eng.probe_attention(0, y) - base).max(axis=1) > 1e-6
    assert changed[9:12].all() and not changed[:9].any() and not changed[12:].any()
    eng.close()


@pytest.mark.parametrize("decay", ["none", "mixed", "instant"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_state_over_extreme_decays(gpu, decay, dtype):
    layer = U.delta(heads=2, kv_heads=1, dim=128, vdim=64, conv=4)
    cfg, w = one_layer(layer, 96, seed=6)
    n = w["l0.mix.dt_bias"].size
    w["l0.mix.dt_bias"] = U.bf16_round({"none": np.full(n, -30.0), "instant": np.full(n, 40.0),
                                        "mixed": np.where(np.arange(n) % 3 == 0, 20.0, np.where(np.arange(n) % 3 == 1, -20.0, -1.0))}[decay])
    w["l0.mix.A_log"] = U.bf16_round(np.full(2, 2.0))
    eng, m = U.engine(gpu, cfg, w, dtype, max_seq_len=512), P.PlainModel(cfg, w)
    x = rows(300, 96)
    want = m.channel_delta("l0.mix.", layer["mixer"], x.astype(np.float64), {})
    U.check(eng.probe_attention(0, x), want, dtype, 2)
    eng.close()


@pytest.mark.parametrize("softcap,scale", [(12.0, 0.7), (3.0, 2.5), (50.0, 1.0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_head_scale_softcap_and_norms(gpu, softcap, scale, dtype):
    cfg = U.config([U.with_ff(U.delta(heads=1, kv_heads=1, dim=8, vdim=8), 24)], width=48, vocab=77, eps=0.1, logit_scale=scale, softcap=softcap)
    w = U.weights(cfg, 2)
    eng, m = U.engine(gpu, cfg, w, dtype), P.PlainModel(cfg, w)
    toks = U.tokens(9, 77)
    got, _ = eng.step([0], [toks], [list(range(9))])
    U.check(got, m.forward(toks, m.new_state()), dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,k,T", [(1, 8, 1), (130, 72, 3), (257, 200, 17), (96, 1000, 65), (640, 136, 300), (129, 64, 129)])
def test_products_of_many_shapes(gpu, n, k, T, dtype):
    """Through a feed-forward whose second matrix is the identity's rows: y = relu(x up^T)^2 padded or cut to the width."""
    cfg, w = one_layer(U.with_ff(U.delta(heads=1, kv_heads=1, dim=8, vdim=8), n), k, seed=n)
    w["l0.mlp.down"] = np.eye(k, n, dtype=np.float32)
    eng, m = U.engine(gpu, cfg, w, dtype, max_seq_len=512), P.PlainModel(cfg, w)
    x = rows(T, k, n)
    U.check(eng.probe_ffn(0, x), m.feed_forward("l0.mlp.", x.astype(np.float64)), dtype)
    eng.close()
