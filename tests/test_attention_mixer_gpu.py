"""Windowed attention over shared key/value heads, alone on the GPU, against the plain implementation."""
import numpy as np
import pytest

import layered_util as U
import plain_mixers as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]

SHAPES = {
    "uneven sizes": (U.attention(), 104),
    "odd sizes": (U.attention(heads=3, kv_heads=3, dim=9, vdim=5, rot_dims=6, window=20, keep_first=3), 41),
    "one dimension per pair": (U.attention(heads=2, kv_heads=1, dim=2, vdim=1, rot_dims=2, window=40, keep_first=1, scale=0.9), 24),
    "large heads, all rotated": (U.attention(heads=8, kv_heads=2, dim=128, vdim=128, rot_dims=128, window=64, keep_first=4, scale=0.09), 256),
    "wide keys, narrow values": (U.attention(heads=4, kv_heads=2, dim=192, vdim=40, rot_dims=64, window=100, keep_first=17, scale=0.07), 128),
    "narrow keys, wide values": (U.attention(heads=4, kv_heads=4, dim=24, vdim=200, rot_dims=24, window=90, keep_first=16), 128),
    "more queries per key than a tile": (U.attention(heads=37, kv_heads=1, dim=16, vdim=16, rot_dims=8, window=65, keep_first=40), 128),
    "window of one": (U.attention(heads=4, kv_heads=2, dim=16, vdim=8, rot_dims=16, window=1, keep_first=0), 64),
    "window of one and kept tokens": (U.attention(heads=4, kv_heads=2, dim=16, vdim=8, rot_dims=16, window=1, keep_first=2), 64),
    "kept tokens past a tile": (U.attention(heads=4, kv_heads=2, dim=16, vdim=104, rot_dims=4, window=16, keep_first=130), 64),
    "window past the context": (U.attention(heads=4, kv_heads=2, dim=32, vdim=32, rot_dims=32, window=5000, keep_first=0), 64),
}


def one_layer(layer, width, seed=1):
    cfg = U.tenetar_config([layer], width=width)
    return cfg, U.tenetar_weights(cfg, seed)


def rows(n, width, seed=0):
    return U.bf16_round(np.random.default_rng(60 + seed).normal(size=(n, width)))


def check_portions(gpu, cfg, w, dtype, sizes, slack=1, page_tokens=16):
    layer, width = cfg["layers"][0], cfg["width"]
    eng, m = U.engine(gpu, cfg, w, dtype, max_seq_len=512, kv_page_tokens=page_tokens), P.plain_model(cfg, w)
    x, states, at = rows(sum(sizes), width), [{}], 0
    for n in sizes:
        want = m.attention(0, x[at : at + n].astype(np.float64), states, at)
        U.check(eng.probe_attention(0, x[at : at + n]), want, dtype, slack)
        at += n
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", SHAPES)
def test_attention_layer(gpu, name, dtype):
    cfg, w = one_layer(*SHAPES[name])
    check_portions(gpu, cfg, w, dtype, (70, 15, 1, 16, 64, 2, 33, 130))  # token by token up to 15 tokens, tiles from 16 on


@pytest.mark.parametrize("page_tokens", [1, 5, 8, 24, 64])
@pytest.mark.parametrize("dims", [(64, 128), (24, 40), (48, 16), (72, 88)])
def test_pages_and_rows_of_other_sizes(gpu, dims, page_tokens):
    """Tiles of keys that end inside pages or span several; cache rows that are swizzled, padded or neither."""
    cfg, w = one_layer(U.attention(heads=4, kv_heads=2, dim=dims[0], vdim=dims[1], rot_dims=16, window=60, keep_first=21, scale=0.1), 64)
    check_portions(gpu, cfg, w, "bfloat16", (70, 1, 1, 40, 3), page_tokens=page_tokens)


@pytest.mark.parametrize("dtype", DTYPES)
def test_no_mask_no_rotation_no_sink(gpu, dtype):
    cfg, w = one_layer(U.attention(window=900, keep_first=0, rot_dims=2, base=1e30), 104)
    w["l0.mix.sink"] = np.full(6, -1e30, np.float32)
    plain = P.plain_model(cfg, w)
    bare = U.tenetar_config([dict(cfg["layers"][0], mixer={k: v for k, v in cfg["layers"][0]["mixer"].items() if k != "mask"})])
    eng = U.engine(gpu, bare, {n: a for n, a in w.items() if n != "l0.mix.sink"}, dtype, max_seq_len=128)
    x = rows(90, 104)
    U.check(eng.probe_attention(0, x), plain.attention(0, x.astype(np.float64), [{}], 0), dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", [-40.0, 0.0, 8.0, 30.0])
def test_sinks_from_nothing_to_everything(gpu, sink, dtype):
    cfg, w = one_layer(U.attention(window=30, keep_first=2), 104)
    w["l0.mix.sink"] = U.bf16_round(sink + np.arange(6) * 0.5)
    check_portions(gpu, cfg, w, dtype, (40, 1, 1, 33))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("eps", [1e-5, 0.5])
def test_norms_span_all_heads(gpu, eps, dtype):
    """One head's projection far larger than the others': a norm per head would make them equal."""
    cfg, w = one_layer(U.attention(), 104)
    cfg["norm"]["eps"] = eps
    w["l0.mix.q"] = w["l0.mix.q"].copy()
    w["l0.mix.q"][:20] *= 8.0
    w["l0.mix.k"] = w["l0.mix.k"].copy()
    w["l0.mix.k"][20:40] *= 8.0
    check_portions(gpu, cfg, w, dtype, (50, 1, 16), 2)


def searching_layer(window, keep_first, seed=7, heads=4, kv_heads=2, dim=40):
    """Rows of kind 1 look for rows of kind 0: queries and keys meet in unrotated dimensions, with a score far above all others."""
    layer = U.attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=16, rot_dims=16, window=window, keep_first=keep_first, scale=0.6)
    cfg, w = one_layer(layer, 96, seed)
    rng = np.random.default_rng(seed)
    ask, key = U.bf16_round(rng.normal(size=96)), U.bf16_round(rng.normal(size=96))
    sign = np.concatenate([np.zeros(16), rng.choice([-1.0, 1.0], dim - 16)])
    for n, count, row in (("q", heads, ask), ("k", kv_heads, key)):
        w["l0.mix." + n] = U.bf16_round(w["l0.mix." + n] + np.tile(np.outer(sign, row / (row @ row)), (count, 1)) * 12.0)
    return cfg, w, ask, key


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep_first", [(16, 0), (37, 5), (64, 16), (65, 17), (128, 1), (200, 70)])
def test_edges_of_window_and_kept_tokens(gpu, window, keep_first, dtype):
    """The one key that is looked for lies just inside or just outside the window, or among or behind the kept first tokens;
    asked for from a prompt's tile and from a token alone."""
    cfg, w, ask, key = searching_layer(window, keep_first)
    m, eng = P.plain_model(cfg, w), U.engine(gpu, cfg, w, dtype, max_seq_len=512)
    n = 330
    base = rows(n, 96, 3)
    shown = 0
    places = sorted({p for p in (0, keep_first - 1, keep_first, keep_first + 1, 15, 16, 63, 64, 100) if 0 <= p < 200})
    for place in places:
        asks = sorted({q for q in (place + 1, place + window - 1, place + window, place + window + 1, place + window + 16, n - 3, n - 1) if place < q < n})
        x = base.copy()
        x[place] = key
        x[asks] = ask
        want = m.attention(0, x.astype(np.float64), [{}], 0)
        lost = x.copy()
        lost[place] = base[5]
        gone = m.attention(0, lost.astype(np.float64), [{}], 0)
        for q in asks:  # the key shows where it is seen, and only there
            seen = q - place < window or place < keep_first
            moved = np.sqrt(np.mean((want[q] - gone[q]) ** 2) / np.mean(want ** 2))
            assert moved > 0.2 if seen else moved < 1e-9
            shown += seen
        eng.kv_clear()
        U.check(eng.probe_attention(0, x)[asks], want[asks], dtype, 2)
        eng.kv_clear()
        out, at = [], 0
        for q in asks:  # everything ahead in one portion, the asking token alone
            if q > at:
                eng.probe_attention(0, x[at:q])
            out.append(eng.probe_attention(0, x[q : q + 1])[0])
            at = q + 1
        U.check(np.array(out), want[asks], dtype, 2)
    assert shown >= len(places)
    eng.close()
