"""The delta rule with separate removal alone on the GPU: step, walk and chunks against the plain implementation."""
import numpy as np
import pytest

import layered_util as U
import plain_mixers as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def rows(n, width, seed=0):
    return U.bf16_round(np.random.default_rng(90 + seed).normal(size=(n, width)))


def model(heads, dim, width, rank=6, seed=1, eps=1e-5, change=None):
    cfg = U.nepudra_config([U.general_delta(heads, dim)], width=width, eps=eps)
    w = U.nepudra_weights(cfg, seed, rank)
    if change:
        change(w)
    return cfg, w, P.plain_model(cfg, w)


def check_cuts(eng, m, x, cuts, dtype, slack=1):
    eng.kv_clear()
    layers, at, got, want = [{}], 0, [], []
    for n in cuts:
        want.append(m.mix(0, x[at : at + n].astype(np.float64), layers, at))
        got.append(eng.probe_attention(0, x[at : at + n]))
        at += n
    U.check(np.concatenate(got), np.concatenate(want), dtype, slack)
    return np.concatenate(got)


SHAPES = {
    "uneven": (3, 20, 104, 6),
    "odd sizes": (2, 9, 41, 3),
    "one channel": (2, 1, 24, 1),
    "exactly a block": (2, 32, 64, 8),
    "a block and one": (1, 33, 40, 5),
    "64": (3, 64, 96, 16),
    "between": (2, 72, 64, 9),
    "128": (2, 128, 128, 24),
    "past the chunked form": (1, 132, 64, 4),
    "256": (1, 256, 64, 7),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", SHAPES)
def test_layer_in_portions(gpu, name, dtype):
    """Runs walked token by token (under 32 tokens), chunks that end on and beside an edge, states carried between them."""
    heads, dim, width, rank = SHAPES[name]
    cfg, w, m = model(heads, dim, width, rank)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=640)
    check_cuts(eng, m, rows(521, width), (32, 1, 31, 33, 2, 63, 64, 65, 1, 97, 4, 128), dtype, 2)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_any_cut_gives_the_same(gpu, dtype):
    cfg, w, m = model(2, 48, 56, 5)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=256)
    x = rows(200, 56, 1)
    whole = check_cuts(eng, m, x, [200], dtype, 2)
    for cuts in ([1] * 200, [2] * 100, [31, 169], [32, 168], [64, 136], [65, 135], [100, 1, 99]):
        U.check(check_cuts(eng, m, x, cuts, dtype, 2), whole, dtype)
    eng.close()


@pytest.mark.parametrize("decay", ["least", "most", "mixed"])
@pytest.mark.parametrize("removal", ["none", "all", "mixed"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_extreme_decays_and_removals(gpu, decay, removal, dtype):
    """Decays at both ends of their range over hundreds of tokens; rates of nothing and everything, also channel by channel."""
    def change(w):
        n = w["l0.mix.w0"].size
        i = np.arange(n)
        w["l0.mix.w0"] = U.bf16_round({"least": np.full(n, -30.0), "most": np.full(n, 30.0), "mixed": np.where(i % 2, 20.0, -20.0)}[decay])
        w["l0.mix.a.b"] = U.bf16_round({"none": np.full(n, -30.0), "all": np.full(n, 30.0), "mixed": np.where(i % 3, 20.0, -20.0)}[removal])
    cfg, w, m = model(2, 64, 96, change=change, seed=3)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=400)
    check_cuts(eng, m, rows(330, 96, 2), [300, 1, 29], dtype, 3)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_that_repeat_and_keys_of_any_length(gpu, dtype):
    """The removed part follows the key's direction, the written part its length: rows of many sizes, whole stretches of one row."""
    def change(w):
        w["l0.mix.a.b"] = np.full_like(w["l0.mix.a.b"], 4.0)
    cfg, w, m = model(2, 32, 64, change=change, seed=4)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=300)
    x = rows(240, 64, 3)
    x[60:130] = x[60]
    x[140:150] *= 8.0
    x[150:160] /= 16.0
    x[170] = 0
    for cuts in ([240], [100, 1, 1, 138], [1] * 40 + [200]):
        check_cuts(eng, m, x, cuts, dtype, 3)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("eps", [1e-5, 0.5])
def test_norm_is_per_head_and_its_weight_is_not(gpu, eps, dtype):
    """One head's values far larger than the other's, and an epsilon that shows."""
    def change(w):
        v = w["l0.mix.v"].copy()
        v[:24] *= 16.0
        w["l0.mix.v"] = v
    cfg, w, m = model(3, 24, 64, eps=eps, change=change)
    eng = U.engine(gpu, cfg, w, dtype)
    x = rows(70, 64, 5)
    check_cuts(eng, m, x, [50, 1, 1, 18], dtype, 2)
    swapped = dict(w, **{"l0.mix.norm": np.roll(w["l0.mix.norm"], 24)})
    assert U.rel_rms(P.plain_model(cfg, swapped).mix(0, x.astype(np.float64), [{}], 0), m.mix(0, x.astype(np.float64), [{}], 0)) > 0.1
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_shows_through_the_state(gpu, dtype):
    """Hardly any decay, no removal, and one token's values far larger than the rest: it shows in every later read-out."""
    def change(w):
        w["l0.mix.w0"] = np.full_like(w["l0.mix.w0"], -12.0)
        w["l0.mix.a.b"] = np.full_like(w["l0.mix.a.b"], -30.0)
    cfg, w, m = model(2, 40, 64, change=change, seed=6)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=400)
    base = rows(300, 64, 4)
    for place in (0, 1, 31, 32, 63, 64, 130):
        x = base.copy()
        x[place] *= 6.0
        want = m.mix(0, x.astype(np.float64), [{}], 0)
        assert U.rel_rms(m.mix(0, base.astype(np.float64), [{}], 0)[-20:], want[-20:]) > 0.3
        for cuts in ([300], [place + 1, 1, 298 - place], [200, 1, 2, 40, 1, 56]):
            check_cuts(eng, m, x, cuts, dtype, 3)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [12, 64, 128])
def test_states_of_many_sequences_step_by_step(gpu, dim, dtype):
    """Decode steps of many slots in no order, sequences that begin among others that go on.  A first token is read as (k . r) v, whose sign
    the norm would bring out however small it is: the epsilon is large enough for what rounding makes of it to stay small."""
    cfg = U.nepudra_config([U.general_delta(4, dim), U.general_delta(2, 16)], width=48, vocab=50, eps=0.05)
    w = U.nepudra_weights(cfg, 5)
    m = P.plain_model(cfg, w)
    n_seqs = 37
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=64, max_seqs=n_seqs)
    slots = np.random.default_rng(1).permutation(n_seqs).tolist()
    lens = [(0, 1, 2, 5, 33, 40)[i % 6] for i in range(n_seqs)]
    toks = [U.tokens(n + 6, 50, 900 + i) for i, n in enumerate(lens)]
    started = [i for i in range(n_seqs) if lens[i]]
    eng.step([slots[i] for i in started], [toks[i][: lens[i]] for i in started], [[] for _ in started])
    looked = [0, 1, 2, 3, 4, 5, 35, 36]
    states = {i: m.new_state() for i in looked}
    for i in looked:
        if lens[i]:
            m.forward(toks[i][: lens[i]], states[i])
    for j in range(6):
        got, _ = eng.step(slots, [[t[n + j]] for t, n in zip(toks, lens)], [[0]] * n_seqs)
        want = np.array([m.forward([toks[i][lens[i] + j]], states[i])[0] for i in looked])
        U.check(got[looked], want, dtype, U.rounding(cfg, dtype))
    eng.close()
