"""Attention with biases, gates per head, factors on queries, bounds, windows and shared caches; token pairs, gated gelu and sums over
depth: each alone on the GPU against the plain implementation."""
import numpy as np
import pytest

import layered_util as U
import plain_mixers as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def rows(n, width, seed=0):
    return U.bf16_round(np.random.default_rng(60 + seed).normal(size=(n, width)))


def model(layer, width=104, seed=1, eps=1e-5, change=None):
    cfg = U.nepudra_config([layer], width=width, eps=eps)
    w = U.nepudra_weights(cfg, seed)
    if change:
        change(w)
    return cfg, w, P.plain_model(cfg, w)


def check_portions(gpu, layer, dtype, sizes, slack=1, page_tokens=16, **kw):
    cfg, w, m = model(layer, **kw)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=640, kv_page_tokens=page_tokens)
    x, layers, at = rows(sum(sizes), cfg["width"]), [{}], 0
    for n in sizes:
        want = m.mix(0, x[at : at + n].astype(np.float64), layers, at)
        U.check(eng.probe_attention(0, x[at : at + n]), want, dtype, slack)
        at += n
    eng.close()


LAYERS = {
    "warm, uneven": U.warm_attention(),
    "warm, odd sizes": U.warm_attention(heads=3, kv_heads=3, dim=9, vdim=5),
    "warm, large heads": U.warm_attention(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.09, temp=(0.3, 64)),
    "warm, wide keys": U.warm_attention(heads=4, kv_heads=2, dim=192, vdim=40, scale=0.07, softcap=None),
    "warm, wide values": U.warm_attention(heads=2, kv_heads=1, dim=24, vdim=200),
    "warm, many queries per key": U.warm_attention(heads=37, kv_heads=1, dim=16, vdim=16, temp=None),
    "warm, one of everything": U.warm_attention(heads=1, kv_heads=1, dim=1, vdim=1, scale=1.0, temp=(2.0, 1)),
    "warm, past the tensor kernels": U.warm_attention(heads=2, kv_heads=1, dim=40, vdim=300),
    "normed, uneven": U.normed_attention(),
    "normed, odd sizes": U.normed_attention(heads=3, kv_heads=3, dim=9, vdim=5, rot_dims=6),
    "normed, large heads": U.normed_attention(heads=8, kv_heads=2, dim=128, vdim=128, rot_dims=128, scale=0.09, window=100, scaling=(4.0, 512, 16.0, 2.0)),
    "normed, shared keys": U.normed_attention(heads=12, kv_heads=3, dim=64, vdim=32, rot_dims=32, window=70),
    "normed, one pair": U.normed_attention(heads=2, kv_heads=1, dim=2, vdim=3, rot_dims=2, scale=0.9, window=5),
    "normed, wide": U.normed_attention(heads=2, kv_heads=1, dim=256, vdim=136, rot_dims=200, scale=0.06, window=33),
    "normed, sees itself alone": U.normed_attention(window=1),
    "normed, two": U.normed_attention(window=2),
    "normed, window past the context": U.normed_attention(window=5000, scaling=None),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", LAYERS)
def test_layer_in_portions(gpu, name, dtype):
    check_portions(gpu, LAYERS[name], dtype, (70, 15, 1, 16, 64, 2, 3, 300, 1, 1))


@pytest.mark.parametrize("page_tokens", [1, 5, 24, 64])
def test_pages_of_other_sizes(gpu, page_tokens):
    for layer in (U.warm_attention(), U.normed_attention()):
        check_portions(gpu, layer, "bfloat16", (70, 1, 1, 40, 3), page_tokens=page_tokens)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("temp", [(3.0, 1), (5.0, 7), (4.0, 64), (2.5, 2.5), (-0.2, 16)])
def test_factors_on_queries(gpu, monkeypatch, temp, dtype):
    """Factors so large that a position off by one would show where they change, in prompts and alone."""
    layer = U.warm_attention(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.4, softcap=None, temp=temp)
    check_portions(gpu, layer, dtype, (66, 1, 1, 1, 1, 57, 1, 2, 16), 2)
    _, _, m = model(layer)
    x, every = rows(130, 104).astype(np.float64), temp[1]
    edges = [p for p in range(20, 130) if np.floor((p + 1) / every) != np.floor(p / every)]
    want = m.mix(0, x, [{}], 0)
    monkeypatch.setattr(P, "query_temperature", lambda pos, t: 1.0 + t["coef"] * np.log(np.floor(np.asarray(pos) / t["every"]) + 1.0))
    moved = U.rel_rms(m.mix(0, x, [{}], 0)[edges], want[edges])
    assert moved > 1e-3  # thirty times the bound in 32-bit


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap", [0.5, 3.0, 50.0, None])
def test_bounded_scores(gpu, cap, dtype):
    layer = U.warm_attention(heads=4, kv_heads=2, dim=32, vdim=16, scale=1.0, softcap=cap, temp=(0.5, 16))
    check_portions(gpu, layer, dtype, (80, 1, 1, 33), 3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [U.warm_attention(), U.normed_attention()])
def test_gates_and_biases(gpu, layer, dtype):
    """Gates per head at half, open or shut; biases that outweigh the projections, and none."""
    for gate, bias in ((0.0, 1.0), (40.0, 1.0), (1.0, 0.0), (1.0, 6.0)):
        def change(w):
            w["l0.mix.g"] = U.bf16_round(w["l0.mix.g"] * gate)
            for n in ("q.b", "k.b", "v.b", "o.b"):
                if "l0.mix." + n in w:
                    w["l0.mix." + n] = U.bf16_round(w["l0.mix." + n] * bias)
        check_portions(gpu, layer, dtype, (20, 1, 17, 2), 2, change=change)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("eps", [1e-5, 0.5])
def test_norms_are_per_head(gpu, eps, dtype):
    def change(w):
        for t in "qk":
            a = w["l0.mix." + t].copy()
            a[:28] *= 16.0
            w["l0.mix." + t] = a
    check_portions(gpu, U.normed_attention(), dtype, (50, 1, 16), 2, eps=eps, change=change)


def searching(kind, dim=40, seed=7, window=37):
    """Rows of kind 1 look for rows of kind 0: queries and keys meet in unrotated dimensions, with a score far above all others."""
    if kind == "warm":
        layer = U.warm_attention(heads=4, kv_heads=2, dim=dim, vdim=16, scale=0.3, softcap=50.0, temp=(0.1, 50))
    else:
        layer = U.normed_attention(heads=4, kv_heads=2, dim=dim, vdim=16, rot_dims=16, scale=1.2, window=window)
    rng = np.random.default_rng(seed)
    ask, key = U.bf16_round(rng.normal(size=96)), U.bf16_round(rng.normal(size=96))
    sign = np.concatenate([np.zeros(16), rng.choice([-1.0, 1.0], dim - 16)])

    def change(w):
        for n, count, row in (("q", 4, ask), ("k", 2, key)):
            w["l0.mix." + n] = U.bf16_round(w["l0.mix." + n] + np.tile(np.outer(sign, row / (row @ row)), (count, 1)) * 4.0)
    return model(layer, 96, seed, change=change) + (ask, key)


def run_asks(eng, x, asks):
    """Everything ahead of an asking row in one portion, the asking row alone."""
    out, at = [], 0
    for q in asks:
        if q > at:
            eng.probe_attention(0, x[at:q])
        out.append(eng.probe_attention(0, x[q : q + 1])[0])
        at = q + 1
    return np.array(out)


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_at_the_edges_of_pages_and_tiles(gpu, dtype):
    cfg, w, m, ask, key = searching("warm")
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=640)
    n, base = 600, rows(600, 96, 3)
    for place in (0, 1, 2, 15, 16, 17, 63, 64, 65, 127, 128, 300, 500):
        asks = sorted({q for q in (place + 1, place + 15, place + 16, place + 63, place + 64, place + 200, n - 3, n - 1) if place < q < n})
        x = base.copy()
        x[place] = key
        x[asks] = ask
        lost = x.copy()
        lost[place] = base[5]
        want = m.mix(0, x.astype(np.float64), [{}], 0)[asks]
        moved = np.sqrt(np.mean((m.mix(0, lost.astype(np.float64), [{}], 0)[asks] - want) ** 2, axis=1) / np.mean(want ** 2))
        assert moved.min() > 0.3, "the far key does not matter: the test would not notice its loss"
        eng.kv_clear()
        U.check(eng.probe_attention(0, x)[asks], want, dtype, 2)
        eng.kv_clear()
        U.check(run_asks(eng, x, asks), want, dtype, 2)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [2, 16, 37, 64, 65, 130])
def test_keys_just_inside_and_just_outside_the_window(gpu, window, dtype):
    """The key that is looked for shows up to window - 1 tokens later and not one more, in prompts, in portions and alone."""
    cfg, w, m, ask, key = searching("normed", window=window)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=640)
    n, base = 420, rows(420, 96, 4)
    for place in (0, 1, 15, 16, 63, 64, 100, 129, 200):
        asks = [place + window - 1, place + window]
        x = base.copy()
        x[asks] = ask
        x[place] = key
        lost = x.copy()
        lost[place] = base[n - 1]
        want = m.mix(0, x.astype(np.float64), [{}], 0)
        gone = m.mix(0, lost.astype(np.float64), [{}], 0)
        moved = np.sqrt(np.mean((gone[asks] - want[asks]) ** 2, axis=1) / np.mean(want[asks] ** 2))
        assert moved[0] > 0.3 and moved[1] < 1e-9, "the window's edge does not show"
        eng.kv_clear()
        U.check(eng.probe_attention(0, x)[asks], want[asks], dtype, 2)
        eng.kv_clear()
        U.check(run_asks(eng, x, asks), want[asks], dtype, 2)
        eng.kv_clear()
        cut = place + window  # the edge between two portions, the second of two tokens
        got = np.concatenate([eng.probe_attention(0, x[:cut]), eng.probe_attention(0, x[cut : cut + 2])])
        U.check(got[asks], want[asks], dtype, 2)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_layer_that_reads_another_layers_keys(gpu, dtype):
    """The second layer's queries look for a key that the first layer wrote, hundreds of tokens back; the first layer is silent."""
    layers = [U.warm_attention(heads=4, kv_heads=2, dim=24, vdim=16, scale=0.3, softcap=60.0, temp=(0.1, 100)),
              U.warm_attention(heads=6, kv_heads=2, dim=24, vdim=16, scale=0.3, softcap=60.0, temp=(0.1, 100), kv_from=0)]
    cfg = U.nepudra_config(layers, width=64, vocab=50)
    w = {k: v.astype(np.float64) for k, v in U.nepudra_weights(cfg, 5).items()}
    w["bigram"] *= 0.05
    for n in ("o", "o.b"):
        w["l0.mix." + n] *= 0.0
    ask, key = w["embed"][1].copy(), w["embed"][0].copy()
    sign = np.random.default_rng(2).choice([-1.0, 1.0], 24)
    w["l1.mix.q"] += np.tile(np.outer(sign, ask / (ask @ ask)), (6, 1)) * 4.0
    w["l0.mix.k"] += np.tile(np.outer(sign, key / (key @ key)), (2, 1)) * 4.0
    w = {n: U.bf16_round(a).reshape(np.shape(a)) for n, a in w.items()}
    m = P.plain_model(cfg, w)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=640)
    n = 600
    for place in (0, 1, 15, 16, 63, 64, 127, 400):
        toks = (2 + np.random.default_rng(place).integers(0, 48, n)).tolist()
        toks[place] = 0
        for q in (place + 1, place + 16, place + 64, n - 2, n - 1):
            toks[q] = 1
        asks = [i for i in range(n) if toks[i] == 1]
        want = m.forward(toks, m.new_state())[asks]
        lost = list(toks)
        lost[place] = 7
        assert U.rel_rms(m.forward(lost, m.new_state())[asks], want) > 0.3, "the far key does not matter"
        eng.kv_clear()
        got, _ = eng.step([0], [toks], [asks])
        U.check(got, want, dtype, 2)
        eng.kv_clear()
        eng.step([0], [toks[: n - 30]], [[]])
        out = [eng.step([0], [[t]], [[0]])[0][0] for t in toks[n - 30 :]]
        late = [i for i in asks if i >= n - 30]
        U.check(np.array([out[i - (n - 30)] for i in late]), want[-len(late) :], dtype, 2)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,width", [(40, 104), (200, 72), (1, 8), (513, 256)])
def test_gated_gelu(gpu, ff, width, dtype):
    cfg, w, m = model(U.with_ff(U.general_delta(1, 8), ff), width)
    eng = U.engine(gpu, cfg, w, dtype)
    x = rows(19, width) * 2
    U.check(eng.probe_ffn(0, x), m.feed_forward(0, x.astype(np.float64)), dtype)
    eng.close()


def quiet(w):
    """Mixers without output: what is left is the embedding, the sums over depth and the head."""
    return {n: np.zeros_like(a) if n.endswith("mix.o") or n.endswith("o.b") else a for n, a in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bigram", [(77, 31, 1009), (1, 3, 5), (4999, 1, 0), (2, 0, 1), (509, 4294967311, 9007199254740881), (131, 1, 1)])
def test_embeddings_of_token_pairs(gpu, bigram, dtype):
    """The pair's row follows the token before, in the same portion or in an earlier one, of the same sequence alone; a first token has a
    row of its own, also when its slot had another sequence before."""
    cfg = U.nepudra_config([U.general_delta(1, 8)], width=24, bigram=bigram)
    w = quiet(U.nepudra_weights(cfg, 3))
    m = P.plain_model(cfg, w)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=128, max_seqs=3)
    V = cfg["vocab"]
    a, b = [5, 5, 0, V - 1, V - 1] + U.tokens(60, V, 1), U.tokens(41, V, 2)
    want_a, want_b = m.forward(a, m.new_state()), m.forward(b, m.new_state())
    got, _ = eng.step([0], [a], [list(range(len(a)))])
    U.check(got, want_a, dtype)
    for cuts in ([1] * 41, [2] * 20 + [1], [40, 1], [1, 39, 1]):
        eng.kv_clear()
        out, at, other = [], 0, 0
        for n in cuts:  # beside another sequence that moves on as well
            ids, parts, want = [2, 1], [b[at : at + n], a[other : other + 1]], [list(range(n)), []]
            got, _ = eng.step(ids, parts, want)
            out.append(got)
            at += n
            other += 1
        U.check(np.concatenate(out), want_b, dtype)
    s = eng.open_sequence()
    for t in (a[:7], b[:3]):
        eng.close_sequence(s)
        s = eng.open_sequence()
        got, _ = eng.step([s], [t], [[0]])
        U.check(got, m.forward(t[:1], m.new_state()), dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [8, 41, 130, 2052, 9000])
def test_sums_over_depth_of_other_widths(gpu, width, dtype):
    """Six layers whose sums weigh every earlier result, some with large or no weight; rows that are no multiple of the vectors, and longer
    than what a block holds in registers."""
    layers = [U.with_ff(U.general_delta(1, 8), 8) if i % 2 else U.general_delta(1, 8) for i in range(6)]
    cfg = U.nepudra_config(layers, width=width, vocab=30, eps=0.05, bigram=(7, 3, 2))
    w = U.nepudra_weights(cfg, 9, depth=0.6)
    w["l2.dwa"] = U.bf16_round(np.array([1.5, 0.0, -0.75, 0.5]))
    w["l4.dwa"] = U.bf16_round(np.array([0.0, 0.5, 0.0, 0.0, 1.0, 0.0]))  # without its own layer's result
    m = P.plain_model(cfg, w)
    eng = U.engine(gpu, cfg, w, dtype)
    toks = U.tokens(23, 30)
    got, _ = eng.step([0], [toks[:20]], [list(range(20))])
    want = m.forward(toks, m.new_state())
    U.check(got, want[:20], dtype, U.rounding(cfg, dtype))
    for i in range(20, 23):
        got, _ = eng.step([0], [[toks[i]]], [[0]])
        U.check(got, want[i : i + 1], dtype, U.rounding(cfg, dtype))
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("eps", [1e-6, 0.3])
def test_norms_of_one_number(gpu, eps, dtype):
    """Gains far from one and an epsilon that shows, on both sublayers and in front of the head."""
    cfg = U.nepudra_config([U.with_ff(U.warm_attention(), 24), U.with_ff(U.general_delta(), 24)], eps=eps)
    w = U.nepudra_weights(cfg, 2)
    for n, g in (("l0.norm1", 0.25), ("l0.norm2", 2.0), ("l1.norm1", -1.5), ("l1.norm2", 0.5), ("final.norm", 3.0)):
        w[n] = np.float32(g).reshape(())
    m = P.plain_model(cfg, w)
    eng = U.engine(gpu, cfg, w, dtype)
    toks = U.tokens(40, cfg["vocab"])
    got, _ = eng.step([0], [toks], [list(range(40))])
    U.check(got, m.forward(toks, m.new_state()), dtype, U.rounding(cfg, dtype))
    eng.close()
