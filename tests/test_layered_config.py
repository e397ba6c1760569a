"""Checkpoint-directory designs without a GPU: the plain implementation against itself, and what the config reader refuses."""
import copy

import numpy as np
import pytest

import layered_util as U
import plain_mixers as P


def mixed_config():
    return U.config([U.with_ff(U.delta(), 40), U.latent(), U.delta(heads=4, kv_heads=2, dim=16, vdim=8, conv=1), U.with_ff(U.latent(heads=2, scaling=None), 56)])


@pytest.mark.parametrize("cuts", [[1] * 23, [2, 5, 1, 9, 6], [22, 1]])
def test_plain_model_in_portions_equals_the_whole(cuts):
    cfg = mixed_config()
    m = P.PlainModel(cfg, U.weights(cfg))
    toks = U.tokens(23, cfg["vocab"])
    whole = m.forward(toks, m.new_state())
    st, parts, at = m.new_state(), [], 0
    for c in cuts:
        parts.append(m.forward(toks[at : at + c], st))
        at += c
    assert np.abs(np.concatenate(parts) - whole).max() < 1e-10


def test_delta_rule_writes_what_it_then_reads():
    """With beta = 1, no decay and a unit key, reading with the key returns the value just written."""
    rng = np.random.default_rng(3)
    k = P.unit(rng.normal(size=(6, 8)), 0.0)
    v = rng.normal(size=(6, 5))
    out = P.delta_rule(k, k, v, np.ones((6, 8)), np.ones(6), np.zeros((8, 5)))
    assert np.allclose(out, v)


def test_causal_convolution_by_definition():
    rng = np.random.default_rng(4)
    x, w = rng.normal(size=(7, 3)), rng.normal(size=(3, 4))
    y, tail = P.causal_conv(x, w, np.zeros((3, 3)))
    for t in range(7):
        want = sum(w[:, 3 - j] * x[t - j] for j in range(4) if t - j >= 0)
        assert np.allclose(y[t], want)
    assert np.allclose(tail, x[-3:])


def test_rotation_preserves_pairs_and_depends_on_distance_only():
    rot = {"dims": 8, "base": 100.0, "scaling": {"factor": 2.0, "original": 32, "fast": 4.0, "slow": 1.0}}
    _, mag = P.yarn_frequencies(rot)
    rng = np.random.default_rng(5)
    q, k = rng.normal(size=(1, 8)), rng.normal(size=(1, 8))
    dots = [float(P.rotate_pairs(q, [p + 9], rot)[0] @ P.rotate_pairs(k, [p], rot)[0]) for p in (0, 3, 50)]
    assert np.allclose(dots, dots[0])
    r = P.rotate_pairs(q, [17], rot)
    assert np.allclose(r[0, ::2] ** 2 + r[0, 1::2] ** 2, (q[0, ::2] ** 2 + q[0, 1::2] ** 2) * mag ** 2)


def test_yarn_leaves_fast_pairs_and_slows_slow_ones():
    base = {"dims": 32, "base": 10000.0}
    f0, m0 = P.yarn_frequencies(base)
    f1, m1 = P.yarn_frequencies(dict(base, scaling={"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}))
    assert m0 == 1.0 and m1 == pytest.approx(0.1 * np.log(4.0) + 1.0)
    assert f1[0] == f0[0] and f1[-1] == pytest.approx(f0[-1] / 4.0)
    assert (f1 <= f0 + 1e-15).all() and (f1 >= f0 / 4.0 - 1e-15).all()


@pytest.mark.parametrize("cuts", [[1] * 60, [2, 5, 1, 9, 6, 37], [58, 2]])
def test_plain_tenetar_in_portions_equals_the_whole(cuts):
    cfg = U.tenetar_mixed()
    m = P.plain_model(cfg, U.tenetar_weights(cfg))
    toks = U.tokens(60, cfg["vocab"])
    whole = m.forward(toks, m.new_state())
    st, parts, at = m.new_state(), [], 0
    for c in cuts:
        parts.append(m.forward(toks[at : at + c], st))
        at += c
    assert np.abs(np.concatenate(parts) - whole).max() < 1e-10


def test_window_and_kept_tokens_by_definition():
    seen = P.visible([0, 3, 9, 10], 11, 4, 2)
    assert [np.flatnonzero(r).tolist() for r in seen] == [[0], [0, 1, 2, 3], [0, 1, 6, 7, 8, 9], [0, 1, 7, 8, 9, 10]]
    assert P.visible([5], 6, 1, 0).sum() == 1 and P.visible([5], 6, 100, 0).all()


def test_sink_is_a_key_without_value():
    """A sink equals one more key whose score is the sink and whose value is zero."""
    rng = np.random.default_rng(2)
    q, k, v = rng.normal(size=(3, 2, 4)), rng.normal(size=(5, 1, 4)), rng.normal(size=(5, 1, 6))
    seen = P.visible([2, 3, 4], 5, 3, 1)
    got = P.sink_attention(q, k, v, 0.5, seen, np.array([0.3, -1.0]))
    for h, sink in enumerate([0.3, -1.0]):
        for t in range(3):
            s = np.append(np.where(seen[t], k[:, 0] @ q[t, h] * 0.5, -np.inf), sink)
            p = np.exp(s - s.max())
            p /= p.sum()
            assert np.allclose(got[t, h], p[:-1] @ v[:, 0])


def test_rotation_of_halves_depends_on_distance_only():
    rng = np.random.default_rng(6)
    q, k = rng.normal(size=(1, 1, 10)), rng.normal(size=(1, 1, 10))
    dots = [float(P.rotate_halves(q, [p + 7], 8, 50.0)[0, 0] @ P.rotate_halves(k, [p], 8, 50.0)[0, 0]) for p in (0, 4, 90)]
    assert np.allclose(dots, dots[0])
    r = P.rotate_halves(q, [3], 8, 50.0)[0, 0]
    assert np.allclose(r[8:], q[0, 0, 8:]) and np.isclose(r[1], q[0, 0, 1] * np.cos(3 * 50.0 ** -0.25) - q[0, 0, 5] * np.sin(3 * 50.0 ** -0.25))


def test_choice_of_experts_by_definition():
    z = np.log(np.array([0.30, 0.02, 0.20, 0.08, 0.25, 0.15]))
    zero = np.zeros(6)
    assert [e for e, _ in P.choose_experts(z, zero, 1, 1, 3)] == [0, 4, 2]
    assert [e for e, _ in P.choose_experts(z, zero, 3, 1, 2)] == [0, 1]
    picks = P.choose_experts(z, np.array([-0.31, 0, 0, 0, 0, 0]), 1, 1, 2)  # the correction moves the choice, not the weight
    assert [e for e, _ in picks] == [4, 2] and np.allclose([s for _, s in picks], [0.25, 0.20])
    low = np.array([-9.0, -9.0, 0, 0, -5.0, -5.0])  # a dropped group loses to negative scores of a kept one
    assert sorted(e for e, _ in P.choose_experts(z, low, 3, 2, 4)) == [2, 3, 4, 5]


@pytest.mark.parametrize("cuts", [[1] * 60, [2, 5, 1, 9, 6, 37], [58, 2]])
def test_plain_munisun_in_portions_equals_the_whole(cuts):
    cfg = U.munisun_mixed()
    m = P.plain_model(cfg, U.munisun_weights(cfg))
    toks = U.tokens(60, cfg["vocab"])
    whole = m.forward(toks, m.new_state())
    st, parts, at = m.new_state(), [], 0
    for c in cuts:
        parts.append(m.forward(toks[at : at + c], st))
        at += c
    assert np.abs(np.concatenate(parts) - whole).max() < 1e-9


def test_frequencies_by_wavelength():
    """Pairs of short wavelength stay, those of long wavelength are stretched by the factor, and the blend is continuous between."""
    rot = {"dims": 64, "base": 10000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}}
    f, g = 10000.0 ** (-np.arange(32) / 32.0), P.wavelength_frequencies(rot)
    turns = 512 * f / (2 * np.pi)
    assert np.allclose(g[turns > 4], f[turns > 4]) and np.allclose(g[turns < 1], f[turns < 1] / 8)
    mid = (turns >= 1) & (turns <= 4)
    assert mid.any() and (turns > 4).any() and (turns < 1).any()
    assert (g[mid] <= f[mid]).all() and (g[mid] >= f[mid] / 8).all() and (np.diff(g) < 0).all()


def test_decayed_sums_by_definition():
    """Token t reads every earlier one with the product of the decays behind it."""
    rng = np.random.default_rng(8)
    q, k, v, d = rng.normal(size=(9, 4)), rng.normal(size=(9, 4)), rng.normal(size=(9, 3)), rng.uniform(0.2, 1.0, 9)
    got = P.decayed_sums(q, k, v, d, np.zeros((4, 3)))
    for t in range(9):
        want = sum((q[t] @ k[s]) * np.prod(d[s + 1 : t + 1]) * v[s] for s in range(t + 1))
        assert np.allclose(got[t], want)


def test_choice_by_sigmoid_by_definition():
    z = np.array([3.0, -4.0, 1.0, 0.9, 0.5, -1.0])
    s = P.sigmoid(z)
    zero = np.zeros(6)
    assert [e for e, _ in P.choose_by_sigmoid(z, zero, 1, 1, 3)] == [0, 2, 3]
    assert [e for e, _ in P.choose_by_sigmoid(z, zero, 3, 1, 2)] == [2, 3]  # the sum of two ranks the groups, not the largest
    picks = P.choose_by_sigmoid(z, np.array([-2.0, 0, 0, 0, 0, 0]), 1, 1, 2)  # the correction moves the choice, not the weight
    assert [e for e, _ in picks] == [2, 3] and np.allclose([v for _, v in picks], s[[2, 3]])
    low = np.array([-9.0, -9.0, -1, -1, -5.0, -5.0])  # a dropped group loses to negative scores of a kept one
    assert sorted(e for e, _ in P.choose_by_sigmoid(z, low, 3, 2, 4)) == [2, 3, 4, 5]


def test_norm_in_parts_and_bounded_scores_by_definition():
    x = np.arange(1.0, 13.0).reshape(2, 6)
    y = P.norm_in_parts(x, 3, 0.5)
    assert np.isclose(y[1, 3], x[1, 3] / np.sqrt((x[1, 2] ** 2 + x[1, 3] ** 2) / 2 + 0.5))
    q, k, v = np.ones((1, 1, 1)), np.array([[[9.0]], [[-9.0]]]), np.array([[[1.0]], [[0.0]]])
    p = P.capped_attention(q, k, v, 1.0, 1, 2.0)[0, 0, 0]
    assert np.isclose(p, 1 / (1 + np.exp(-2 * 2 * np.tanh(4.5))))


@pytest.mark.parametrize("cuts", [[1] * 60, [2, 5, 1, 9, 6, 37], [58, 2]])
def test_plain_nepudra_in_portions_equals_the_whole(cuts):
    cfg = U.nepudra_mixed()
    m = P.plain_model(cfg, U.nepudra_weights(cfg))
    toks = U.tokens(60, cfg["vocab"])
    whole = m.forward(toks, m.new_state())
    st, parts, at = m.new_state(), [], 0
    for c in cuts:
        parts.append(m.forward(toks[at : at + c], st))
        at += c
    assert np.abs(np.concatenate(parts) - whole).max() < 1e-9


def test_general_delta_rule_by_definition():
    """Without removal it is a decayed sum; with full removal and no decay a repeated unit key replaces what it wrote before."""
    rng = np.random.default_rng(9)
    r, k, v = rng.normal(size=(7, 5)), rng.normal(size=(7, 5)), rng.normal(size=(7, 5))
    w = rng.uniform(0.5, 1.0, (7, 5))
    got = P.general_delta_rule(r, k, v, w, np.zeros((7, 5)), np.zeros((5, 5)))
    for t in range(7):
        want = sum((r[t] * np.prod(w[s + 1 : t + 1], axis=0)) @ k[s] * v[s] for s in range(t + 1))
        assert np.allclose(got[t], want)
    key = np.tile(P.unit(k[:1], 0.0), (7, 1))
    assert np.allclose(P.general_delta_rule(key, key, v, np.ones((7, 5)), np.ones((7, 5)), np.zeros((5, 5)), 0.0), v)
    # removal and decay both look at the state before the token
    S, u = rng.normal(size=(5, 5)), P.unit(k[0])
    want = np.diag(w[0]) @ S - np.outer(0.3 * u, u @ S) + np.outer(k[0], v[0])
    assert np.allclose(P.general_delta_rule(r[:1], k[:1], v[:1], w[:1], np.full((1, 5), 0.3), S.copy())[0], want.T @ r[0])


def test_query_temperature_and_token_pairs_by_definition():
    f = P.query_temperature(np.arange(9), {"coef": 0.5, "every": 4})
    assert np.allclose(f, [1, 1, 1] + [1 + 0.5 * np.log(2)] * 4 + [1 + 0.5 * np.log(3)] * 2)
    rows = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert P.pair_rows([4, 5, 0], None, rows) == [10, (12 + 35) % 10, 5] and P.pair_rows([4], 5, rows) == [(15 + 28) % 10]


def test_rotation_of_half_pairs_takes_the_scaled_frequencies():
    rot = {"dims": 8, "base": 50.0, "scaling": {"factor": 4.0, "original": 32, "fast": 4.0, "slow": 1.0}}
    f, mag = P.yarn_frequencies(rot)
    x = np.random.default_rng(1).normal(size=(1, 1, 11))
    y = P.rotate_half_pairs(x, [5], rot)[0, 0]
    assert np.allclose(y[8:], x[0, 0, 8:]) and np.isclose(y[1], mag * (x[0, 0, 1] * np.cos(5 * f[1]) - x[0, 0, 5] * np.sin(5 * f[1])))
    plain = {"dims": 8, "base": 50.0}
    assert np.allclose(P.rotate_half_pairs(x, [5], plain), P.rotate_halves(x, [5], 8, 50.0))


def broken_nepudra(change):
    cfg = copy.deepcopy(U.nepudra_mixed())
    change(cfg)
    return cfg


@pytest.mark.parametrize("change,text", [
    (lambda c: c["embedding"].pop("bigram"), "bigram"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda c: c["embedding"]["bigram"].update(mul_cur=1.5), "factor"),
    (lambda c: c["layers"][0].update(type="channel_delta"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1), "softcap"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=30), "rotated"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=0), "cannot read"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=4), "earlier"),
    (lambda c: c["layers"][6]["mixer"].update(kv_from=4), "cannot read"),
    (lambda c: c["layers"][6]["mlp"].update(kind="moe"), "unknown kind"),
])
def test_nepudra_config_errors_are_named(lc, change, text):
    with pytest.raises(lc.LeafcutterError) as e:
        lc.Engine.from_config(broken_nepudra(change))
    assert text in str(e.value)


def broken_munisun(change):
    cfg = copy.deepcopy(U.munisun_mixed())
    change(cfg)
    return cfg


@pytest.mark.parametrize("change,text", [
    (lambda c: c.pop("token_side"), "token_side"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c["layers"][0].update(type="attention"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"]["right"]["decay"].__setitem__(0, 1.5), "decay"),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(softcap=0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("high"), "high"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(groups=4), "key heads"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][1]["mlp"].update(shared={"ff": 8}), "shared"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
])
def test_munisun_config_errors_are_named(lc, change, text):
    with pytest.raises(lc.LeafcutterError) as e:
        lc.Engine.from_config(broken_munisun(change))
    assert text in str(e.value)


def broken_tenetar(change):
    cfg = copy.deepcopy(U.tenetar_mixed())
    change(cfg)
    return cfg


@pytest.mark.parametrize("change,text", [
    (lambda c: c.pop("embedding"), "embedding"),
    (lambda c: c["layers"][0].update(type="channel_delta"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "key heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), "rotated"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "cannot read"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=3), "cannot read"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
])
def test_tenetar_config_errors_are_named(lc, change, text):
    with pytest.raises(lc.LeafcutterError) as e:
        lc.Engine.from_config(broken_tenetar(change))
    assert text in str(e.value)


def broken(change):
    cfg = copy.deepcopy(mixed_config())
    change(cfg)
    return cfg


@pytest.mark.parametrize("change,text", [
    (lambda c: c.update(architecture="Nobody"), "not known"),
    (lambda c: c.pop("architecture"), "architecture"),
    (lambda c: c.update(width=0), "width"),
    (lambda c: c.update(width=10.5), "width"),
    (lambda c: c.update(layers=[]), "no layers"),
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=2), "key heads"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "unknown kind"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "odd"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), "rotated"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_config_errors_are_named(lc, change, text):
    with pytest.raises(lc.LeafcutterError) as e:
        lc.Engine.from_config(broken(change))
    assert text in str(e.value)


def test_missing_files_are_errors(lc, tmp_path):
    with pytest.raises(lc.LeafcutterError) as e:
        lc.Engine.load_dir(str(tmp_path))
    assert "config.json" in str(e.value)


def test_bf16_tensors_from_the_generator(lc):
    """The generator's bf16 values are its f32 values rounded to nearest even."""
    from leafcutterllm_b200 import synth
    f = synth.host_tensor(lc.TYPE_F32, 7, "t", 4096).view(np.float32)
    b = synth.host_tensor(lc.TYPE_BF16, 7, "t", 4096).view(np.uint16)
    assert np.array_equal(b, U.bf16_bytes(f))


def test_command_line_inspects_a_checkpoint_directory(lc, tmp_path, capsys):
    from leafcutterllm_b200.__main__ import main
    cfg = mixed_config()
    U.write_checkpoint(tmp_path, cfg, U.weights(cfg))
    assert main(["inspect", "--model", str(tmp_path)]) == 0
    import json
    assert json.loads(capsys.readouterr().out) == {"architecture": "Varasun", "width": 104, "vocab": 131, "layers": {"channel_delta": 2, "latent_attention": 2}}
    assert main(["generate", "--model", str(tmp_path / "nothing"), "--tokens", "1,2"]) == 1
    assert "error" in capsys.readouterr().err
