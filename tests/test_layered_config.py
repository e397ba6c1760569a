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
