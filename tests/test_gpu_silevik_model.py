"""The sandwich-normed design's own mechanisms in whole models (the tests shared with the other designs are in test_gpu_hybrid_model.py):
the residual stream layer by layer, the reach of a window, sinks, value mixing, what a layer may leave out, refusals."""
import json

import numpy as np
import pytest

import hybrid_models as H
import silevik_models as S
from ingot_b200 import models as M

pytestmark = pytest.mark.gpu


def open_model(tmp, cfg, w, **kw):
    return M.Model(H.write(tmp, cfg, w), **kw)


def three_kinds(**kw):
    return S.config([S.layer("attention", 4, 2, 24, 16, 21, rot=10, mlp=S.dense(40)), S.layer("attention_2", 6, 2, 12, 16, mlp=S.moe(4, 2, 6, None, 24, 16)),
                     S.layer("attention_3", 2, 2, 16, 16, rot=16, scaling=(2.0, 32, 4.0, 1.0), mlp=S.moe(3, 0, 3, (1, 1), 16, 24))], vocab=70, width=52, **kw)


@pytest.mark.parametrize("f32", [True, False])
def test_residual_stream_after_every_layer(tmp_path, f32):
    cfg = three_kinds()
    w = S.random_weights(cfg, 4)
    t = np.random.default_rng(0).integers(0, 70, 90).tolist()
    want = []
    S.reference_logits(cfg, w, t, want)
    with open_model(tmp_path, cfg, w, f32=f32, max_tokens=128) as m:
        m.tap()
        m.step([(0, 0, t[:80], [79])])
        whole = m.residuals().reshape(3, 80, 52)
        for p in range(80, 90):
            m.step([(0, p, t[p:p + 1], [0])])
        single = m.residuals().reshape(10, 3, 52).transpose(1, 0, 2)
    for g, x in zip(np.concatenate([whole, single], axis=1), want):
        assert np.abs(g - x).max() < (1e-5 if f32 else 4e-2) * np.abs(x).max()


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("window", [1, 15, 16, 17, 40, 64])
def test_reach_of_a_window(tmp_path, window, f32, decoded):
    """One layer: changing token j moves the logits at j + window - 1 and leaves those at j + window exactly as they were."""
    cfg = S.config([S.layer("attention", 4, 2, 16, 12, window, rot=8, scale=0.03)], vocab=60, width=40)
    w = S.random_weights(cfg, window)
    t = np.random.default_rng(1).integers(0, 60, 120).tolist()
    with open_model(tmp_path, cfg, w, f32=f32, max_tokens=128) as m:
        def logits(tokens):
            cut = 20 if decoded else 120
            out = [m.step([(0, 0, tokens[:cut], list(range(cut)))])] + [m.step([(0, p, tokens[p:p + 1], [0])]) for p in range(cut, 120)]
            m.release(0)
            return np.concatenate(out)
        base = logits(t)
        for j in (0, 15, 16, 31, 47):
            other = list(t)
            other[j] = (t[j] + 7) % 60
            moved = np.abs(logits(other) - base).max(axis=1)
            assert not moved[:j].any() and not moved[j + window:].any()
            assert (moved[j:j + window] > 1e-6).all()


@pytest.mark.parametrize("least", ["1", "300", "1000000"])
def test_the_kernel_a_portion_takes_does_not_show(tmp_path, monkeypatch, least):
    """Portions of all sizes of several sequences beside single tokens, on either kernel or on both in turn, against the plain implementation."""
    monkeypatch.setenv("INGOT_GQA_LONG", least)
    cfg = S.config([S.layer("attention", 6, 2, 40, 24, 90, rot=20, scale=0.15, mlp=S.dense(40)), S.layer("attention_2", 3, 1, 72, 48, scale=0.1, v_mix=False),
                    S.layer("attention_3", 4, 2, 16, 24, rot=8, mlp=S.moe(3, 2, 5, None, 24, 16))], vocab=40, width=44)
    w = S.random_weights(cfg, 4)
    rng = np.random.default_rng(0)
    tokens = [rng.integers(0, 40, n).tolist() for n in (600, 330, 150)]
    want = [S.reference_logits(cfg, w, t) for t in tokens]
    with open_model(tmp_path, cfg, w, max_tokens=1152, max_seqs=3, max_step_tokens=320) as m:
        at, got = [0, 0, 0], [[], [], []]
        cuts = [[150, 2, 100, 1, 180, 3, 64], [40, 1, 39, 130, 120], [1, 2, 41, 100, 6]]
        for k in range(40):
            step = []
            for s in range(3):
                n = min(cuts[s][k % len(cuts[s])], len(tokens[s]) - at[s])
                if n > 0:
                    step.append((s, at[s], tokens[s][at[s]:at[s] + n], list(range(n))))
            if not step:
                break
            rows, r = m.step(step), 0
            for s, p, t, _ in step:
                got[s].append(rows[r:r + len(t)])
                r += len(t)
                at[s] += len(t)
        assert at == [600, 330, 150]
        for s in range(3):
            assert H.error(np.concatenate(got[s]), want[s]).max() < 4e-2, s


def test_a_far_key_decides(tmp_path):
    """Layers that see everything: one token hundreds of positions back has a score far above all others, for a portion and for decoded
    tokens; taking it away shows."""
    cfg = S.config([S.layer("attention_2", 2, 1, 16, 16, scale=1.0), S.layer("attention_3", 2, 1, 16, 16, rot=2, base=1e6, scale=1.0)], vocab=40, width=32)
    w = S.random_weights(cfg, 3)
    rng = np.random.default_rng(2)
    t = rng.integers(2, 40, 700).tolist()
    t[5] = 1  # the only one of its kind
    w["embed"][1] = 0
    w["embed"][1, 0] = M.from_bf16(M.to_bf16(np.float32([8.0])))[0]
    for layer in (0, 1):
        k = w[f"l{layer}.mix.k"]
        k[:, 0] = 4.0  # its keys answer to the first coordinate
        w[f"l{layer}.mix.k.norm"][:] = 1.5
    want = S.reference_logits(cfg, w, t)
    other = list(t)
    other[5] = 2
    assert H.error(S.reference_logits(cfg, w, other), want)[650:].max() > 0.1
    for f32, tol in ((True, 3e-5), (False, 4e-2)):
        with open_model(tmp_path, cfg, w, f32=f32, max_tokens=704) as m:
            got = [m.step([(0, 0, t[:300], list(range(300)))]), m.step([(0, 300, t[300:690], list(range(390)))])]
            got += [m.step([(0, p, t[p:p + 1], [0])]) for p in range(690, 700)]
        assert H.error(np.concatenate(got), want).max() < tol


def test_values_are_mixed_with_the_first_mixing_layers(tmp_path):
    """The first layer that mixes gives its values and ignores its own weight; layers that do not mix keep out of it. Portions and slots in
    any order: nothing of it outlives a step."""
    layers = [S.layer("attention_2", 2, 2, 8, 12, v_mix=False), S.layer("attention", 4, 2, 8, 12, 9, rot=4), S.layer("attention_2", 2, 1, 8, 20, v_mix=False),
              S.layer("attention_3", 2, 2, 8, 12, rot=4)]
    cfg = S.config(layers, vocab=50, width=32)
    w = S.random_weights(cfg, 2)
    rng = np.random.default_rng(3)
    a, b = rng.integers(0, 50, 40).tolist(), rng.integers(0, 50, 33).tolist()
    wa, wb = S.reference_logits(cfg, w, a), S.reference_logits(cfg, w, b)
    changed = dict(w)
    changed["l1.mix.vmix"] = w["l1.mix.vmix"] * 0.5
    assert np.array_equal(S.reference_logits(cfg, changed, a), wa)
    changed["l3.mix.vmix"] = w["l3.mix.vmix"] * 0.5
    assert H.error(S.reference_logits(cfg, changed, a), wa).max() > 1e-3
    with open_model(tmp_path, cfg, w, f32=True, max_tokens=128, max_seqs=2) as m:
        got_a, got_b = [], []
        for at_a, n_a, at_b, n_b in ((0, 7, 0, 2), (7, 2, 2, 20), (9, 30, 22, 1), (39, 1, 23, 10)):
            rows = m.step([(1, at_b, b[at_b:at_b + n_b], list(range(n_b))), (0, at_a, a[at_a:at_a + n_a], list(range(n_a)))])
            got_b.append(rows[:n_b])
            got_a.append(rows[n_b:])
        assert H.error(np.concatenate(got_a), wa).max() < 3e-5 and H.error(np.concatenate(got_b), wb).max() < 3e-5


def test_pages_behind_the_window_serve_other_sequences(tmp_path):
    """Windowed layers beside layers that see everything, three sequences that together fill the pool; what is released is used again."""
    cfg = S.config([S.layer("attention", 2, 1, 16, 16, 20, rot=4, mlp=S.dense(16)), S.layer("attention_2", 2, 1, 16, 16)], vocab=40, width=24)
    w = S.random_weights(cfg, 6)
    t = np.random.default_rng(2).integers(0, 40, 320).tolist()
    want = S.reference_logits(cfg, w, t)
    with open_model(tmp_path, cfg, w, f32=True, max_tokens=960, max_seqs=3, max_step_tokens=32) as m:
        for again in range(2):
            got = {s: [] for s in range(3)}
            for p in range(0, 320, 10):
                rows = m.step([(s, p, t[p:p + 10], list(range(10))) for s in range(3)])
                for s in range(3):
                    got[s].append(rows[s * 10:s * 10 + 10])
            for s in range(3):
                assert H.error(np.concatenate(got[s]), want).max() < 3e-5
                m.release(s)


@pytest.mark.parametrize("f32", [True, False])
def test_single_tokens_on_the_streaming_kernels(tmp_path, f32):
    """Widths the weight-streaming products of single tokens take, experts and shared expert included."""
    cfg = S.config([S.layer("attention", 8, 2, 32, 64, 40, rot=16, mlp=S.dense(512)), S.layer("attention_2", 4, 2, 64, 64, mlp=S.moe(3, 1, 4, (2, 2), 256, 256))], vocab=300, width=256)
    w = S.random_weights(cfg, 9)
    t = np.random.default_rng(5).integers(0, 300, 70).tolist()
    want = S.reference_logits(cfg, w, t)
    with open_model(tmp_path, cfg, w, f32=f32, max_tokens=128, max_seqs=2) as m:
        got = np.concatenate([m.step([(0, 0, t[:3], [0, 1, 2])])] + [m.step([(0, p, t[p:p + 1], [0])]) for p in range(3, 70)])
    assert H.error(got, want).max() < (3e-5 if f32 else 4e-2)


def test_constants_come_from_the_configuration(tmp_path):
    cfg = three_kinds()
    w = S.random_weights(cfg, 1)
    t = np.random.default_rng(4).integers(0, 70, 60).tolist()
    base = S.reference_logits(cfg, w, t)

    def changed(path, value):
        c = json.loads(json.dumps(cfg))
        at = c
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        return c
    for i, (path, value) in enumerate([(("logit_scale",), 1.25), (("embedding", "scale"), 0.5), (("norm", "eps"), 0.3), (("layers", 0, "mixer", "scale"), 0.6),
                                       (("layers", 0, "mixer", "rot", "base"), 50.0), (("layers", 0, "mixer", "rot", "dims"), 24), (("layers", 0, "mixer", "mask", "size"), 5),
                                       (("layers", 2, "mixer", "rot", "scaling", "factor"), 6.0), (("layers", 2, "mixer", "rot", "scaling", "original"), 300),
                                       (("layers", 2, "mixer", "rot", "scaling", "fast"), 1.5), (("layers", 2, "mixer", "rot", "scaling", "slow"), 0.1),
                                       (("layers", 1, "mlp", "router", "scale"), 4.0), (("layers", 1, "mlp", "router", "top"), 2), (("layers", 1, "mixer", "v_mix"), False)]):
        c = changed(path, value)
        want = S.reference_logits(c, w, t)
        assert H.error(want, base).max() > 1e-4, path
        with open_model(tmp_path / str(i), c, w, f32=True, max_tokens=64) as m:
            assert H.error(m.step([(0, 0, t, list(range(60)))]), want).max() < 5e-5, path


def test_refusals(tmp_path):
    cfg = three_kinds()
    w = S.random_weights(cfg)

    def refused(change, text, name):
        c = json.loads(json.dumps(cfg))
        change(c)
        with pytest.raises(M.ModelError, match=text):
            open_model(tmp_path / name, c, w)
    mixer = lambda c, i: c["layers"][i]["mixer"]
    refused(lambda c: mixer(c, 0)["rot"].update(dims=7), "even", "a")
    refused(lambda c: mixer(c, 0)["rot"].update(dims=26), "more than", "b")
    refused(lambda c: mixer(c, 0).update(kv_heads=3), "multiple", "c")
    refused(lambda c: c["layers"][1]["mlp"]["router"].update(groups={"count": 4, "keep": 1}), "equal groups", "d")
    refused(lambda c: c["layers"][1]["mlp"]["router"].update(groups={"count": 2, "keep": 1}), "kept groups", "e")
    refused(lambda c: mixer(c, 2).update(kv_heads=1), "shape", "f")
    refused(lambda c: c["layers"][2].update(type="attention_4"), "unknown layer type", "g")
    missing = {k: v for k, v in w.items() if k != "l2.mix.sink"}
    with pytest.raises(M.ModelError, match="sink is missing"):
        open_model(tmp_path / "h", cfg, missing)
    two = S.config([S.layer("attention_2", 2, 2, 8, 12), S.layer("attention_2", 2, 1, 8, 24)], vocab=20, width=16)
    with pytest.raises(M.ModelError, match="mix values"):
        open_model(tmp_path / "i", two, S.random_weights(two))
