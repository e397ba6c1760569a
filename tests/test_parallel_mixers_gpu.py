"""Attention beside a linear recurrence, each branch and their meeting alone on the GPU, against the plain implementation."""
import numpy as np
import pytest

import layered_util as U
import plain_mixers as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def rows(n, width, seed=0):
    return U.bf16_round(np.random.default_rng(80 + seed).normal(size=(n, width)))


def model(layer, width=104, seed=1, only=None, eps=1e-5, change=None):
    """only: 'left' or 'right': the other branch's output matrix is zero."""
    cfg = U.munisun_config([layer], width=width, eps=eps)
    w = U.munisun_weights(cfg, seed)
    if only:
        drop = "l0.mix.%s.o" % ("right" if only == "left" else "left")
        w[drop] = np.zeros_like(w[drop])
    if change:
        change(w)
    return cfg, w


def check_portions(gpu, cfg, w, dtype, sizes, slack=1, page_tokens=16, seed=0):
    eng, m = U.engine(gpu, cfg, w, dtype, max_seq_len=640, kv_page_tokens=page_tokens), P.plain_model(cfg, w)
    x, st, at = rows(sum(sizes), cfg["width"], seed), {}, 0
    for n in sizes:
        want = m.mix(0, x[at : at + n].astype(np.float64), st, at)
        U.check(eng.probe_attention(0, x[at : at + n]), want, dtype, slack)
        at += n
    eng.close()


ATTENTION = {
    "gated, uneven": U.scaled_pair(U.gated_attention()),
    "gated, odd sizes": U.scaled_pair(U.gated_attention(heads=3, kv_heads=3, dim=9, vdim=5, rot_dims=6)),
    "gated, large heads": U.scaled_pair(U.gated_attention(heads=8, kv_heads=2, dim=128, vdim=128, rot_dims=128, scale=0.09, softcap=20.0)),
    "gated, wide keys": U.scaled_pair(U.gated_attention(heads=4, kv_heads=2, dim=192, vdim=40, rot_dims=64, scale=0.07)),
    "gated, wide values": U.scaled_pair(U.gated_attention(heads=2, kv_heads=1, dim=24, vdim=200, rot_dims=24, softcap=None)),
    "gated, many queries per key": U.scaled_pair(U.gated_attention(heads=37, kv_heads=1, dim=16, vdim=16, rot_dims=8)),
    "convolved, uneven": U.normed_pair(U.conv_attention()),
    "convolved, odd sizes": U.normed_pair(U.conv_attention(heads=3, kv_heads=3, dim=9, vdim=5, rot_dims=6, conv=4)),
    "convolved, one dimension per pair": U.normed_pair(U.conv_attention(heads=2, kv_heads=1, dim=2, vdim=1, rot_dims=2, conv=2, scale=0.9)),
    "convolved, large heads": U.normed_pair(U.conv_attention(heads=4, kv_heads=4, dim=128, vdim=128, rot_dims=64, conv=4, scale=0.09)),
    "convolved, wide": U.normed_pair(U.conv_attention(heads=2, kv_heads=1, dim=256, vdim=136, rot_dims=200, conv=3, scale=0.06)),
    "convolved, past the tensor kernels": U.normed_pair(U.conv_attention(heads=2, kv_heads=1, dim=40, vdim=300, rot_dims=40, conv=2)),
    "convolved, one tap": U.normed_pair(U.conv_attention(conv=1)),
    "convolved, many taps": U.normed_pair(U.conv_attention(conv=7)),
    "convolved, capped and slowed": U.normed_pair(U.conv_attention(softcap=2.0, scaling=(8.0, 1.0, 4.0, 60), rot_dims=20)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ATTENTION)
def test_attention_branch(gpu, name, dtype):
    cfg, w = model(ATTENTION[name], only="left")
    check_portions(gpu, cfg, w, dtype, (70, 15, 1, 16, 64, 2, 3, 300, 1, 1), U.rounding(cfg, dtype))


@pytest.mark.parametrize("page_tokens", [1, 5, 24, 64])
def test_pages_of_other_sizes(gpu, page_tokens):
    for layer in (U.scaled_pair(), U.normed_pair()):
        cfg, w = model(layer)
        check_portions(gpu, cfg, w, "bfloat16", (70, 1, 1, 40, 3), page_tokens=page_tokens)


SPACES = {
    "uneven": (U.state_space(), 104),
    "one group": (U.state_space(heads=5, groups=1, state=32, vdim=24, norm_groups=1), 72),
    "a group per head": (U.state_space(heads=4, groups=4, state=16, vdim=40, conv=2, norm_groups=8), 64),
    "norm parts across heads": (U.state_space(heads=4, groups=2, state=8, vdim=24, conv=3, norm_groups=3), 64),
    "odd sizes": (U.state_space(heads=3, groups=3, state=9, vdim=7, conv=5, norm_groups=3), 41),
    "one tap": (U.state_space(conv=1), 40),
    "large state": (U.state_space(heads=2, groups=1, state=256, vdim=64, norm_groups=2), 128),
    "large": (U.state_space(heads=4, groups=2, state=128, vdim=128, norm_groups=4), 256),
    "more value columns than a block": (U.state_space(heads=2, groups=2, state=64, vdim=104, norm_groups=1), 96),
    "state padded": (U.state_space(heads=2, groups=2, state=40, vdim=32, norm_groups=2), 96),
}
LIGHTNINGS = {
    "uneven": (U.lightning(), 104),
    "odd sizes": (U.lightning((0.5, 0.97, 0.9), dim=7, vdim=11), 41),
    "one head": (U.lightning((0.999,), dim=64, vdim=16), 72),
    "large": (U.lightning((0.7, 0.99, 0.9999, 0.1), dim=128, vdim=128), 256),
    "wide keys": (U.lightning((0.9, 0.999), dim=256, vdim=32), 64),
    "wide values": (U.lightning((0.9, 0.95), dim=24, vdim=264), 64),
    "extremes": (U.lightning((0.0, 1.0, 1e-30), dim=32, vdim=24), 64),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SPACES) + ["lightning " + n for n in LIGHTNINGS])
def test_recurrent_branch(gpu, name, dtype):
    """Runs walked token by token (under 32 tokens), runs in chunks that end on and beside a chunk's edge, states carried between both."""
    if name.startswith("lightning "):
        right, width = LIGHTNINGS[name[10:]]
        layer = U.normed_pair(right=right)
    else:
        right, width = SPACES[name]
        layer = U.scaled_pair(right=right)
    cfg, w = model(layer, width, only="right")
    check_portions(gpu, cfg, w, dtype, (64, 1, 31, 32, 2, 33, 63, 65, 1, 129, 5, 128), 2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decay", ["none", "instant", "mixed", "bursts"])
def test_states_over_extreme_decays(gpu, decay, dtype):
    """Steps and decays from nothing to everything; bursts: a few tokens forget all that came before them, in the middle of chunks whose
    other tokens keep nearly everything."""
    def change(w):
        a, b = "l0.mix.right.A_log", "l0.mix.right.dt_bias"
        n = w[a].size
        w[a] = U.bf16_round({"none": np.full(n, -20.0), "instant": np.full(n, 4.0), "mixed": np.linspace(-8, 4, n), "bursts": np.full(n, 3.0)}[decay])
        if decay == "bursts":
            w[b] = U.bf16_round(np.full(n, -9.0))
            w["l0.mix.right.in"][-n:] = U.bf16_round(np.tile(direction / 4, (n, 1)))
    direction = np.random.default_rng(3).choice([-1.0, 1.0], 96)
    layer = U.scaled_pair(right=U.state_space(heads=4, groups=2, state=64, vdim=32, norm_groups=2))
    cfg, w = model(layer, 96, only="right", change=change)
    eng, m = U.engine(gpu, cfg, w, dtype, max_seq_len=512), P.plain_model(cfg, w)
    x = rows(330, 96)
    if decay == "bursts":
        x[[40, 41, 100, 191, 192, 250]] = U.bf16_round(direction)
    want = m.mix(0, x.astype(np.float64), {}, 0)
    U.check(eng.probe_attention(0, x), want, dtype, 2)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer,tensors", [(U.normed_pair(U.conv_attention(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2, conv=3)), ("left.v.conv",)),
                                           (U.scaled_pair(right=U.state_space(heads=1, groups=1, state=8, vdim=8, conv=3, norm_groups=1)), ("right.conv",))])
def test_convolutions_reach_exactly_taps_tokens_back(gpu, layer, tensors, dtype):
    """Only the oldest tap weighs: taking one input row away changes what depends on it from taps - 1 rows later on, also across calls."""
    only = "left" if tensors[0].startswith("left") else "right"
    def change(w):
        for t in tensors:
            c = np.zeros_like(w["l0.mix." + t])
            c[:, 0] = 1.0
            w["l0.mix." + t] = c
        if only == "left":  # every token looks at itself alone
            for t in "qk":
                w["l0.mix.left." + t] = np.tile(w["l0.mix.left." + t][:1] * 0, (8, 1))
        else:  # a state that forgets at once
            w["l0.mix.right.A_log"] = np.full(1, 9.0, np.float32)
            w["l0.mix.right.dt_bias"] = np.full(1, 5.0, np.float32)
    cfg, w = model(layer, 32, only=only, change=change)
    eng, m = U.engine(gpu, cfg, w, dtype), P.plain_model(cfg, w)
    x = rows(44, 32)
    y = x.copy()
    y[9] = 0
    for cuts in ([44], [9, 1, 34], [10, 1, 1, 32], [8, 3, 33]):
        both = []
        for z in (x, y):
            eng.kv_clear()
            at, out = 0, []
            for c in cuts:
                out.append(eng.probe_attention(0, z[at : at + c]))
                at += c
            both.append(np.concatenate(out))
            U.check(both[-1], m.mix(0, z.astype(np.float64), {}, 0), dtype, 2)
        moved = np.abs(both[0] - both[1]).max(axis=1) > 1e-6
        assert moved[11] and not moved[:9].any() and not (only == "right" and moved[12:].any())
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [U.scaled_pair(), U.normed_pair()])
@pytest.mark.parametrize("eps", [1e-5, 0.5])
def test_norms_are_per_head(gpu, layer, eps, dtype):
    """One head's projections far larger than the others', and an epsilon that shows."""
    def change(w):
        for t, n in (("q", 1), ("k", 1)):
            a = w["l0.mix.left." + t].copy()
            a[: layer["mixer"]["left"]["dim"] * n] *= 16.0
            w["l0.mix.left." + t] = a
    cfg, w = model(layer, only="left", eps=eps, change=change)
    check_portions(gpu, cfg, w, dtype, (50, 1, 16), 2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap", [0.5, 3.0, 50.0, None])
def test_bounded_scores(gpu, cap, dtype):
    """Scores far above the bound: without it the largest would take all the weight."""
    cfg, w = model(U.scaled_pair(U.gated_attention(heads=4, kv_heads=2, dim=32, vdim=16, rot_dims=32, scale=2.0, softcap=cap)), only="left")
    check_portions(gpu, cfg, w, dtype, (80, 1, 1, 33), 2)
    if cap == 3.0:
        m = P.plain_model(cfg, w)
        x = rows(60, 104).astype(np.float64)
        bare = P.plain_model(dict(cfg, layers=[U.scaled_pair(dict(cfg["layers"][0]["mixer"]["left"], softcap=1e6))]), w)
        assert U.rel_rms(bare.mix(0, x, {}, 0), m.mix(0, x, {}, 0)) > 0.3


@pytest.mark.parametrize("dtype", DTYPES)
def test_output_gate(gpu, dtype):
    for gain in (0.0, 40.0):
        def change(w):
            w["l0.mix.left.g"] = U.bf16_round(w["l0.mix.left.g"] * gain)
        cfg, w = model(U.scaled_pair(), only="left", change=change)
        check_portions(gpu, cfg, w, dtype, (20, 1, 17), 2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_both_branches_meet(gpu, dtype):
    for layer in (U.scaled_pair(left_scale=1.0, right_scale=1.0), U.scaled_pair(left_scale=-0.3, right_scale=2.5), U.normed_pair()):
        cfg, w = model(layer)
        check_portions(gpu, cfg, w, dtype, (40, 1, 2, 90, 17))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [8, 41, 130, 2052, 9000])
def test_sums_of_normed_branches_of_other_widths(gpu, width, dtype):
    """Rows that are no multiple of the vectors, and longer than what a block holds in registers."""
    cfg, w = model(U.normed_pair(U.conv_attention(heads=2, kv_heads=1, dim=8, vdim=8, rot_dims=4), U.lightning((0.9,), dim=8, vdim=8)), width)
    check_portions(gpu, cfg, w, dtype, (3, 1), 2)


def searching_model(kind, seed=7, dim=40):
    """Rows of kind 1 look for rows of kind 0: queries and keys meet in unrotated dimensions, with a score far above all others."""
    heads, kv_heads = 4, 2
    if kind == "gated":
        layer = U.scaled_pair(U.gated_attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=16, rot_dims=16, scale=1.2, softcap=50.0, scaling=(4.0, 1.0, 4.0, 64)))
    else:
        layer = U.normed_pair(U.conv_attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=16, rot_dims=16, scale=1.2, conv=3))
    rng = np.random.default_rng(seed)
    ask, key = U.bf16_round(rng.normal(size=96)), U.bf16_round(rng.normal(size=96))
    sign = np.concatenate([np.zeros(16), rng.choice([-1.0, 1.0], dim - 16)])

    def change(w):
        for n, count, row in (("q", heads, ask), ("k", kv_heads, key)):
            w["l0.mix.left." + n] = U.bf16_round(w["l0.mix.left." + n] + np.tile(np.outer(sign, row / (row @ row)), (count, 1)) * 4.0)
            if kind != "gated":  # the current token outweighs its neighbours
                c = w["l0.mix.left.%s.conv" % n] * 0.1
                c[:, -1] = 1.0
                w["l0.mix.left.%s.conv" % n] = U.bf16_round(c)
    cfg, w = model(layer, 96, seed, only="left", change=change)
    return cfg, w, ask, key


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["gated", "convolved"])
def test_far_keys_at_the_edges_of_pages_and_tiles(gpu, kind, dtype):
    """The one key that is looked for, in the prompt; asked for from a prompt's tile and from a token alone."""
    cfg, w, ask, key = searching_model(kind)
    m, eng = P.plain_model(cfg, w), U.engine(gpu, cfg, w, dtype, max_seq_len=640)
    n = 600
    base = rows(n, 96, 3)
    for place in (0, 1, 2, 15, 16, 17, 63, 64, 65, 127, 128, 300, 500):
        asks = sorted({q for q in (place + 1, place + 15, place + 16, place + 63, place + 64, place + 200, n - 3, n - 1) if place < q < n})
        x = base.copy()
        x[place] = key
        x[asks] = ask
        want = m.mix(0, x.astype(np.float64), {}, 0)
        lost = x.copy()
        lost[place] = base[5]
        moved = np.sqrt(np.mean((m.mix(0, lost.astype(np.float64), {}, 0)[asks] - want[asks]) ** 2, axis=1) / np.mean(want[asks] ** 2))
        assert moved.min() > 0.5, "the far key does not matter: the test would not notice its loss"
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
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["space", "lightning"])
def test_a_far_token_shows_through_the_state(gpu, kind, dtype):
    """Nothing decays and one token carries values sixteen times larger than the rest: it shows in every later read-out, through
    chunks, single steps and portions."""
    if kind == "space":
        layer = U.scaled_pair(right=U.state_space(heads=8, groups=8, state=16, vdim=16, norm_groups=1))
        change = lambda w: w.update({"l0.mix.right.A_log": np.full(8, -20.0, np.float32)})
    else:
        layer, change = U.normed_pair(right=U.lightning((1.0,) * 8, dim=16, vdim=16)), None
    cfg, w = model(layer, 64, only="right", change=change)
    m, eng = P.plain_model(cfg, w), U.engine(gpu, cfg, w, dtype, max_seq_len=640)
    base = rows(300, 64, 4)
    for place in (0, 31, 63, 64, 130):
        x = base.copy()
        x[place] *= 16.0
        want = m.mix(0, x.astype(np.float64), {}, 0)
        assert U.rel_rms(m.mix(0, base.astype(np.float64), {}, 0)[-20:], want[-20:]) > 0.3
        for cuts in ([300], [place + 1, 1, 298 - place], [200, 1, 2, 40, 1, 56]):
            eng.kv_clear()
            at, out = 0, []
            for c in cuts:
                out.append(eng.probe_attention(0, x[at : at + c]))
                at += c
            U.check(np.concatenate(out)[place + 1 :], want[place + 1 :], dtype, max(2, U.rounding(cfg, dtype)))
    eng.close()


def quiet(cfg, w):
    """Mixers without output: what is left is the embedding, the token inputs and the head."""
    for n in w:
        if n.endswith("left.o") or n.endswith("right.o"):
            w[n] = np.zeros_like(w[n])
    return w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("side,width", [(1, 24), (11, 41), (24, 104), (130, 64)])
def test_token_inputs_of_every_layer(gpu, side, width, dtype):
    cfg = U.munisun_config([U.scaled_pair(), U.normed_pair(), U.with_ff(U.scaled_pair(), 24)], width=width, side=side)
    w = quiet(cfg, U.munisun_weights(cfg, side))
    m, eng = P.plain_model(cfg, w), U.engine(gpu, cfg, w, dtype)
    toks = [5, 5, 0, cfg["vocab"] - 1] + U.tokens(30, cfg["vocab"])
    got, _ = eng.step([0], [toks], [list(range(34))])
    want = m.forward(toks, m.new_state())
    U.check(got, want, dtype)
    one, _ = eng.step([0], [[7]], [[0]])
    st = m.new_state()
    U.check(one, m.forward([7], st), dtype)  # nothing carries over when no mixer speaks
    swapped = dict(w, **{"side.embed": np.roll(w["side.embed"], side, axis=1)})
    assert U.rel_rms(P.plain_model(cfg, swapped).forward(toks, m.new_state()), want) > 0.2
    eng.close()
