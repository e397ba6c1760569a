"""Checkpoint-directory models through the engine's step, cache, slots, batches and generation, against the plain model."""
import io
import json
import sys

import numpy as np
import pytest

import layered_util as U
import plain_mixers as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def mixed_config():
    return U.config([U.with_ff(U.delta(), 40), U.latent(), U.delta(heads=4, kv_heads=2, dim=16, vdim=8, conv=3),
                     U.with_ff(U.latent(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=48, q_rank=20, scaling=None), 56)])


@pytest.fixture(scope="module", params=["varasun", "tenetar", "munisun", "nepudra"])
def model(request):
    if request.param == "varasun":
        cfg = mixed_config()
        w = U.weights(cfg, 11)
    elif request.param == "munisun":
        cfg = U.munisun_mixed()
        w = U.munisun_weights(cfg, 13, fixed_choice=True)
    elif request.param == "nepudra":
        cfg = U.nepudra_mixed()
        w = U.nepudra_weights(cfg, 14)
    else:
        cfg = U.tenetar_mixed()
        w = U.tenetar_weights(cfg, 12, fixed_choice=True)
    return cfg, w, P.plain_model(cfg, w)


def run_cut(eng, slot, toks, cuts):
    out, at = [], 0
    for c in cuts:
        logits, _ = eng.step([slot], [toks[at : at + c]], [list(range(c))])
        out.append(logits)
        at += c
    assert at == len(toks)
    return np.concatenate(out)


def portions(n, sizes):
    cuts, i = [], 0
    while sum(cuts) < n:
        cuts.append(min(sizes[i % len(sizes)], n - sum(cuts)))
        i += 1
    return cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[300], [1], [2], [3, 1, 2], [16], [15, 17], [64, 65], [100, 7], [129, 2]])
def test_prompts_in_portions(gpu, model, sizes, dtype):
    cfg, w, m = model
    n = 300 if sizes[0] > 3 else 70
    toks = U.tokens(n, cfg["vocab"], n)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=320)
    want = m.forward(toks, m.new_state())
    U.check(run_cut(eng, 0, toks, portions(n, sizes)), want, dtype, U.rounding(cfg, dtype))
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(gpu, model, dtype):
    cfg, w, m = model
    eng = U.engine(gpu, cfg, w, dtype)
    for n in (1, 2, 3, 4, 5):
        for cuts in ([n], [1] * n):
            eng.kv_clear()
            toks = U.tokens(n, cfg["vocab"], 70 + n)
            U.check(run_cut(eng, 0, toks, cuts), m.forward(toks, m.new_state()), dtype, U.rounding(cfg, dtype))
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("design", ["varasun", "tenetar", "munisun", "nepudra"])
def test_a_call_longer_than_one_pass(gpu, design, dtype):
    """More tokens in one call than a pass takes (2048): the second pass continues from the first one's cache and state."""
    if design == "varasun":
        cfg = U.config([U.delta(heads=1, kv_heads=1, dim=16, vdim=16, conv=4), U.latent(heads=2, dim=8, rot_dim=8, vdim=8, kv_rank=24, q_rank=16)], width=32, vocab=40)
        w = U.weights(cfg, 3)
    elif design == "munisun":
        cfg = U.munisun_config([U.with_gated_experts(U.scaled_pair(U.gated_attention(heads=2, kv_heads=1, dim=8, vdim=8, rot_dims=4), U.state_space(heads=2, groups=1, state=16, vdim=8)),
                                                     experts=6, top=2, groups=3, keep=2),
                                U.normed_pair(U.conv_attention(heads=2, kv_heads=1, dim=8, vdim=8), U.lightning((0.9, 0.999), dim=8, vdim=8))], width=32, vocab=40)
        w = U.munisun_weights(cfg, 3, fixed_choice=True)
    elif design == "nepudra":
        cfg = U.nepudra_config([U.general_delta(heads=2, dim=16), U.warm_attention(heads=2, kv_heads=1, dim=8, vdim=8, temp=(0.3, 500)),
                                U.normed_attention(heads=2, kv_heads=1, dim=8, vdim=8, rot_dims=4, window=700)], width=32, vocab=40)
        w = U.nepudra_weights(cfg, 3)
    else:
        cfg = U.tenetar_config([U.with_experts(U.attention(heads=2, kv_heads=1, dim=8, vdim=8, window=700, keep_first=70), experts=5, identity=1, top=2, groups=2, keep=1),
                                U.attention(heads=2, kv_heads=1, dim=8, vdim=8, window=3000, keep_first=0, kv_from=0)], width=32, vocab=40)
        w = U.tenetar_weights(cfg, 3, fixed_choice=True)
    m = P.plain_model(cfg, w)
    a, b = U.tokens(1500, 40, 1), U.tokens(703, 40, 2)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=2304, max_seqs=2)
    got, _ = eng.step([0, 1], [a, b], [[0, 1499], [546, 547, 548, 549, 702]])
    want = np.concatenate([m.forward(a, m.new_state())[[0, 1499]], m.forward(b, m.new_state())[[546, 547, 548, 549, 702]]])
    U.check(got, want, dtype, U.rounding(cfg, dtype))
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batches_equal_each_alone(gpu, model, dtype):
    """Portions of prompts beside single decoded tokens, sequences left out of steps, wanted rows in any number."""
    cfg, w, m = model
    lens = [90, 23, 151, 5]
    toks = [U.tokens(n, cfg["vocab"], 20 + n) for n in lens]
    want = [m.forward(t, m.new_state()) for t in toks]
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=160, max_seqs=4)
    plan = [[(0, 40), (2, 1)], [(2, 64), (0, 1), (1, 20)], [(1, 1), (3, 2)], [(0, 1), (1, 1), (2, 17), (3, 1)], [(2, 1), (0, 47)], [(3, 2), (1, 1), (0, 1), (2, 68)]]
    at = [0] * 4
    for step in plan:
        ids = [s for s, _ in step]
        parts = [toks[s][at[s] : at[s] + n] for s, n in step]
        places = [list(range(0, n, 2)) if s != 1 else [] for s, n in step]
        got, nxt = eng.step(ids, parts, places)
        exp = np.concatenate([want[s][[at[s] + p for p in pl]] for (s, n), pl in zip(step, places)])
        U.check(got, exp, dtype, U.rounding(cfg, dtype))
        assert (nxt == got.argmax(axis=1)).all()
        for s, n in step:
            at[s] += n
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_are_used_again(gpu, model, dtype):
    """A pool for 128 tokens and two slots serve many sequences one after the other; nothing of an earlier one shows."""
    cfg, w, m = model
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=128, max_seqs=2, kv_pool_tokens=128)
    rng = np.random.default_rng(8)
    live = {}
    for i in range(14):
        while len(live) == 2 or (live and rng.random() < 0.4):
            eng.close_sequence(live.pop(next(iter(live))))
        s = eng.open_sequence()
        live[i] = s
        n = int(rng.integers(1, 64))
        toks = U.tokens(n, cfg["vocab"], 200 + i)
        cuts = portions(n, [int(rng.integers(1, 33)), 1, 2])
        U.check(run_cut(eng, s, toks, cuts), m.forward(toks, m.new_state()), dtype, U.rounding(cfg, dtype))
    eng.close()


@pytest.mark.parametrize("sizes", [[260], [1], [2, 70], [33, 1, 1, 2]])
@pytest.mark.parametrize("design", ["tenetar", "munisun"])
def test_choices_that_follow_the_token(gpu, design, sizes):
    """Every token its own experts (in 32-bit, where rounding does not move a choice): portions, then other sequences beside it."""
    cfg = U.tenetar_mixed() if design == "tenetar" else U.munisun_mixed()
    w = U.tenetar_weights(cfg, 21) if design == "tenetar" else U.munisun_weights(cfg, 21)
    m = P.plain_model(cfg, w)
    toks = U.tokens(260, cfg["vocab"], 9)
    want = m.forward(toks, m.new_state())
    eng = U.engine(gpu, cfg, w, "float32", max_seq_len=272, max_seqs=3)
    U.check(run_cut(eng, 0, toks, portions(260, sizes)), want, "float32")
    eng.kv_clear()
    other = U.tokens(90, cfg["vocab"], 10)
    beside = m.forward(other, m.new_state())
    eng.step([1, 2], [other[:40], toks[:100]], [[], []])
    got, _ = eng.step([2, 1, 0], [toks[100:], other[40:41], toks[:9]], [[0, 159], [0], [8]])
    U.check(got, np.concatenate([want[[100, 259]], beside[[40]], want[[8]]]), "float32")
    eng.close()


def test_slots_and_pool_run_out_loudly(gpu, model):
    cfg, w, _ = model
    eng = U.engine(gpu, cfg, w, max_seq_len=128, max_seqs=2, kv_pool_tokens=64)
    a, b = eng.open_sequence(), eng.open_sequence()
    assert a != b
    with pytest.raises(gpu.LeafcutterError) as e:
        eng.open_sequence()
    assert e.value.status == -5
    eng.step([a], [U.tokens(40, cfg["vocab"])], [[]])
    with pytest.raises(gpu.LeafcutterError) as e:
        eng.step([b], [U.tokens(40, cfg["vocab"])], [[]])
    assert e.value.status == -5
    eng.close_sequence(a)
    eng.step([b], [U.tokens(40, cfg["vocab"])], [[39]])
    with pytest.raises(gpu.LeafcutterError):
        eng.step([b], [[1, 2]], [[2]])
    with pytest.raises(gpu.LeafcutterError):
        eng.close_sequence(a)
    eng.close()


def far_key_model(seed=5):
    """One attention layer in which token 1 looks for token 0: its query has one outstanding score with token 0's key."""
    layer = U.latent(heads=3, dim=24, rot_dim=8, vdim=16, kv_rank=40, q_rank=32, scale=0.2, scaling=(2.0, 64, 8.0, 1.0))
    cfg = U.config([layer], width=64, vocab=50)
    w = {k: v.astype(np.float64) for k, v in U.weights(cfg, seed).items()}
    eps, mx = cfg["norm"]["eps"], layer["mixer"]
    cq = P.rms_norm(w["l0.mix.dq"] @ w["embed"][1], eps, w["l0.mix.dq.norm"])
    c = P.rms_norm((w["l0.mix.dkv"] @ w["embed"][0])[: mx["kv_rank"]], eps, w["l0.mix.dkv.norm"])
    D, R = mx["dim"], mx["rot_dim"]
    for h in range(mx["heads"]):
        k = w["l0.mix.uk"][h * D : (h + 1) * D] @ c
        w["l0.mix.uq"][h * (D + R) : h * (D + R) + D] += np.outer(k / (k @ k), cq / (cq @ cq)) * 60.0  # a score of 12 above the rest
    return cfg, {n: U.bf16_round(a) for n, a in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_show_in_prompts_and_in_decoding(gpu, dtype):
    cfg, w = far_key_model()
    m = P.PlainModel(cfg, w)
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=1100)
    n = 1040
    for place in (0, 1, 15, 16, 17, 63, 64, 127, 128, 511, 1000):
        toks = (2 + np.random.default_rng(place).integers(0, 48, n)).tolist()
        toks[place] = 0
        for q in (place + 1, place + 15, place + 16, place + 48, place + 64, 700, 1022, n - 2, n - 1):
            if place < q < n:
                toks[q] = 1
        asks = [i for i in range(n) if toks[i] == 1]
        want = m.forward(toks, m.new_state())[asks]
        lost = list(toks)
        lost[place] = 7
        assert U.rel_rms(m.forward(lost, m.new_state())[asks], want) > 0.3, "the far key does not matter: the test would not notice its loss"
        eng.kv_clear()
        got, _ = eng.step([0], [toks], [asks])
        U.check(got, want, dtype, 2)
        eng.kv_clear()
        eng.step([0], [toks[: n - 30]], [[]])
        out = [eng.step([0], [[t]], [[0]])[0][0] for t in toks[n - 30 :]]
        late = [i for i in asks if i >= n - 30]
        U.check(np.array([out[i - (n - 30)] for i in late]), want[-len(late) :], dtype, 2)
    eng.close()


def test_long_decoding_and_greedy_generation(gpu, model):
    """generate(), the callback path, the device-resident loop and a batch of sequences give the plain model's greedy tokens."""
    cfg, w, m = model
    eng = U.engine(gpu, cfg, w, "float32", max_seq_len=512, max_seqs=3)
    prompts = [U.tokens(n, cfg["vocab"], 400 + n) for n in (19, 3, 40)]
    ref = []  # the plain model's tokens, up to the first pick between two logits that rounding could swap
    for p in prompts:
        st = m.new_state()
        row, out = m.forward(p, st)[-1], []
        while len(out) < 220:
            first, second = np.sort(row)[[-1, -2]]
            if first - second < 1e-4:
                break
            out.append(int(row.argmax()))
            row = m.forward([out[-1]], st)[-1]
        ref.append(out)
    assert min(len(r) for r in ref) >= 60 and max(len(r) for r in ref) == 220
    assert eng.generate(prompts[0], 220, stop_on_eos=False)[: len(ref[0])] == ref[0]
    seen = []
    eng.generate(prompts[1], 60, stop_on_eos=False, on_token=seen.append)
    assert seen == ref[1][:60]
    eng.kv_clear()
    _, nxt = eng.forward_batch([0, 1, 2], prompts, want_logits=False)
    toks, _ = eng.decode_loop([0, 1, 2], nxt, 100)
    for i in range(3):
        n = min(len(ref[i]), 101)
        assert ([int(nxt[i])] + toks[:, i].tolist())[:n] == ref[i][:n]
    assert eng.counters()["tokens_decoded"] >= 300 and eng.kv_memory_bytes() > 0
    # seeded sampling runs through the same path and repeats
    a = eng.generate(prompts[0], 20, temperature=0.8, top_p=0.9, seed=3, stop_on_eos=False)
    assert a == eng.generate(prompts[0], 20, temperature=0.8, top_p=0.9, seed=3, stop_on_eos=False)
    eng.close()


@pytest.mark.parametrize("n_seqs", [1, 5, 20, 70])
@pytest.mark.parametrize("design", ["varasun", "tenetar", "munisun", "nepudra"])
def test_decode_batches_of_every_product_form(gpu, design, n_seqs):
    """Decode steps whose token count selects different tiles, at contexts on both sides of page and key-tile edges."""
    if design == "varasun":
        cfg = U.config([U.with_ff(U.delta(heads=2, kv_heads=1, dim=64, vdim=64), 136), U.latent(heads=20, dim=32, rot_dim=16, vdim=32, kv_rank=96, q_rank=64)], width=128)
        w = U.weights(cfg, 4)
    elif design == "munisun":
        cfg = U.munisun_config([U.with_ff(U.scaled_pair(U.gated_attention(heads=20, kv_heads=2, dim=32, vdim=32), U.state_space(heads=4, groups=2, state=64, vdim=64)), 136),
                                U.with_gated_experts(U.normed_pair(U.conv_attention(heads=20, kv_heads=2, dim=32, vdim=32), U.lightning((0.9, 0.999, 0.5), dim=64, vdim=32)),
                                                     experts=8, top=3, groups=4, keep=3, ff=130)], width=128, side=40)
        w = U.munisun_weights(cfg, 4, fixed_choice=True)
    elif design == "nepudra":
        cfg = U.nepudra_config([U.with_ff(U.warm_attention(heads=20, kv_heads=2, dim=32, vdim=32, temp=(0.5, 20)), 136), U.general_delta(heads=4, dim=64),
                                U.with_ff(U.warm_attention(heads=20, kv_heads=2, dim=32, vdim=32, kv_from=0), 72),
                                U.normed_attention(heads=12, kv_heads=3, dim=64, vdim=32, rot_dims=64, window=64)], width=128)
        w = U.nepudra_weights(cfg, 4)
    else:
        cfg = U.tenetar_config([U.with_ff(U.attention(heads=20, kv_heads=2, dim=32, vdim=32, window=64, keep_first=16), 136),
                                U.with_experts(U.attention(heads=20, kv_heads=2, dim=32, vdim=32, window=150, keep_first=0, kv_from=0), experts=6, identity=2, top=3, groups=4,
                                               keep=3, ff=130, shared_ff=64)], width=128)
        w = U.tenetar_weights(cfg, 4, fixed_choice=True)
    m = P.plain_model(cfg, w)
    eng = U.engine(gpu, cfg, w, "bfloat16", max_seq_len=200, max_seqs=n_seqs)
    lens = [(1, 15, 16, 17, 63, 64, 65, 127, 129)[i % 9] for i in range(n_seqs)]
    toks = [U.tokens(n + 3, cfg["vocab"], 700 + i) for i, n in enumerate(lens)]
    eng.step(list(range(n_seqs)), [t[:n] for t, n in zip(toks, lens)], [[] for _ in lens])
    for j in range(3):
        got, _ = eng.step(list(range(n_seqs)), [[t[n + j]] for t, n in zip(toks, lens)], [[0]] * n_seqs)
        want = np.array([m.forward(t[: n + j + 1], m.new_state())[-1] for t, n in zip(toks[:10], lens)])
        U.check(got[:10], want, "bfloat16", U.rounding(cfg, "bfloat16"))
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_checkpoint_directory_and_trace_runner(gpu, model, tmp_path, monkeypatch, capsys, dtype):
    from leafcutterllm_b200 import Engine, trace
    cfg, w, m = model
    U.write_checkpoint(tmp_path, cfg, w)
    eng = Engine.load_dir(str(tmp_path), max_seq_len=64, dtype=dtype)
    toks = U.tokens(33, cfg["vocab"], 5)
    want = m.forward(toks, m.new_state())
    U.check(eng.forward(toks)[None], want[-1:], dtype, U.rounding(cfg, dtype))
    eng.close()
    from leafcutterllm_b200.__main__ import main
    st, picks = m.new_state(), []
    line = m.forward(toks, st)[-1]
    for _ in range(4):
        picks.append(int(line.argmax()))
        line = m.forward(picks[-1:], st)[-1]
    assert main(["generate", "--model", str(tmp_path), "--tokens", ",".join(map(str, toks)), "--max-tokens", "4", "--dtype", "float32", "--keep-going"]) == 0
    assert [int(t) for t in capsys.readouterr().out.split()] == picks
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:20], "want": [19, 3]}, {"id": "y", "tokens": toks[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[1:3], "want": []}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "z", "tokens": toks, "want": [32]}, {"id": "x", "tokens": toks[20:21], "want": [0]}], "end": ["x", "z"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    out = tmp_path / "out"
    out.mkdir()
    assert trace.main(["--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "192"]) == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1", "done", "2"]
    got = np.fromfile(out / "0.f32", "<f4").reshape(2, -1)
    U.check(got, want[[19, 3]], dtype, U.rounding(cfg, dtype))
    assert not (out / "1.f32").exists()
    got = np.fromfile(out / "2.f32", "<f4").reshape(2, -1)
    U.check(got, want[[32, 20]], dtype, U.rounding(cfg, dtype))


def test_incomplete_models_are_named(gpu, model):
    cfg, w, _ = model
    dropped = {"Tenetar": ("l1.mlp.e3.down", "l2.mlp.correction", "l0.norm1b", "l3.mix.q.norm"), "Varasun": ("l1.mix.uk", "l0.mix.a1"),
               "Munisun": ("l0.mix.left.k.conv", "l1.mix.right.conv.b", "l1.mix.left.g", "l2.mlp.e9.gate", "l3.side.norm", "side.embed", "l0.mix.right.out"),
               "Nepudra": ("bigram", "l0.mix.w1", "l0.mix.a.b", "l1.mix.k.b", "l1.mix.g", "l1.mix.o.b", "l2.mix.k.norm", "l3.norm2", "l4.dwa", "l4.mix.q.b")}[cfg["architecture"]]
    for drop, status in [(n, -6) for n in dropped + ("final.norm",)]:
        with pytest.raises(gpu.LeafcutterError) as e:
            U.engine(gpu, cfg, {n: a for n, a in w.items() if n != drop})
        assert e.value.status == status and drop in str(e.value)
    wrong = dict(w)
    name = {"Tenetar": "l2.mlp.e1.up", "Varasun": "l1.mix.uv", "Munisun": "l1.mix.right.in", "Nepudra": "l3.mix.w2"}[cfg["architecture"]]
    wrong[name] = w[name][:-1]
    with pytest.raises(gpu.LeafcutterError) as e:
        U.engine(gpu, cfg, wrong)
    assert e.value.status == -1 and name in str(e.value)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [dict(heads=8, groups=2, state=16, vdim=8, conv=4), dict(heads=16, groups=16, state=64, vdim=64, conv=2), dict(heads=12, groups=4, state=40, vdim=24, conv=3)])
def test_states_of_many_sequences_step_by_step(gpu, shape, dtype):
    """Decode steps of so many states that they pass through a ring of copies; new sequences among them, slots in no order."""
    heads, dim, vdim = shape["heads"], shape["state"], shape["vdim"]
    small = U.conv_attention(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2)
    cfg = U.munisun_config([U.scaled_pair(U.gated_attention(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2), U.state_space(norm_groups=2, **shape)),
                            U.normed_pair(small, U.lightning(tuple(1.0 - 0.9 ** h for h in range(heads)), dim=dim, vdim=vdim))], width=48, vocab=50)
    w = U.munisun_weights(cfg, 5)
    m = P.plain_model(cfg, w)
    n_seqs = 75
    eng = U.engine(gpu, cfg, w, dtype, max_seq_len=64, max_seqs=n_seqs)
    slots = np.random.default_rng(1).permutation(n_seqs).tolist()
    lens = [(0, 1, 2, 5, 33, 40)[i % 6] for i in range(n_seqs)]
    toks = [U.tokens(n + 6, 50, 900 + i) for i, n in enumerate(lens)]
    started = [i for i in range(n_seqs) if lens[i]]
    eng.step([slots[i] for i in started], [toks[i][: lens[i]] for i in started], [[] for _ in started])
    looked = [0, 1, 2, 3, 4, 5, 36, 70, 73, 74]
    states = {i: m.new_state() for i in looked}
    for i in looked:
        if lens[i]:
            m.forward(toks[i][: lens[i]], states[i])
    for j in range(6):
        got, _ = eng.step(slots, [[t[n + j]] for t, n in zip(toks, lens)], [[0]] * n_seqs)
        want = np.array([m.forward([toks[i][lens[i] + j]], states[i])[0] for i in looked])
        U.check(got[looked], want, dtype, U.rounding(cfg, dtype))
    eng.close()
