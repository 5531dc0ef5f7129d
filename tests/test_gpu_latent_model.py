"""The latent / mixture design's own mechanisms in whole models (the tests shared with the other designs are in
test_gpu_hybrid_model.py): the residual stream layer by layer, the reach of a window, state that outlives a portion, refusals."""
import json

import numpy as np
import pytest

import hybrid_models as H
import latent_moe_models as L
from ingot_b200 import models as M

pytestmark = pytest.mark.gpu


def open_model(tmp, cfg, w, **kw):
    return M.Model(H.write(tmp, cfg, w), **kw)


@pytest.mark.parametrize("f32", [True, False])
def test_residual_stream_after_every_layer_run(tmp_path, f32):
    cfg = L.config([L.layer(3, 10, 6, 14, 21, 9, experts=4, top=4, ff=20), L.layer(2, 8, 4, 8, 24, 30)], vocab=40, width=44, loop=(0, 1, 3), bigram=(23, 9, 5))
    w = L.random_weights(cfg, 4)
    t = np.random.default_rng(0).integers(0, 40, 41).tolist()
    want = []
    L.reference_logits(cfg, w, t, want)
    with open_model(tmp_path, cfg, w, f32=f32, max_tokens=64) as m:
        m.tap()
        m.step([(0, 0, t, [40])])
        got = m.residuals().reshape(len(want), 41, 44)
    assert len(want) == 4
    for g, x in zip(got, want):
        assert np.abs(g - x).max() < (2e-5 if f32 else 6e-2) * np.abs(x).max()


@pytest.mark.parametrize("least", [0, 2, 40])
def test_portions_on_the_rows_and_on_the_expansion_agree(tmp_path, monkeypatch, least):
    """The length from which portions run on expanded keys does not show: portions of all sizes of several sequences in one step, more
    keys than are expanded at a time, against the plain implementation."""
    monkeypatch.setenv("INGOT_LATENT_EXPAND", str(least))
    cfg = L.config([L.layer(3, 10, 6, 14, 21, 30, experts=4, top=4, ff=20), L.layer(2, 72, 8, 100, 40, 200, scale=0.1), L.layer(3, 10, 6, 14, 21, 30)], vocab=40, width=44,
                   loop=(1, 3, 2), bigram=(23, 9, 5))
    w = L.random_weights(cfg, 4)
    rng = np.random.default_rng(0)
    tokens = [rng.integers(0, 40, n).tolist() for n in (600, 330, 150)]
    want = [L.reference_logits(cfg, w, t) for t in tokens]
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


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("window", [1, 15, 16, 17, 40])
def test_reach_of_a_window(tmp_path, window, f32, decoded):
    """One layer: changing token j moves the logits at j + window - 1 and leaves those at j + window exactly as they were."""
    cfg = L.config([L.layer(2, 8, 8, 12, 24, window, scale=0.04, experts=3, top=3, ff=16)], vocab=60, width=40)
    w = L.random_weights(cfg, window)
    t = np.random.default_rng(1).integers(0, 60, 100).tolist()
    with open_model(tmp_path, cfg, w, f32=f32, max_tokens=128) as m:
        def logits(tokens):
            cut = 20 if decoded else 100
            out = [m.step([(0, 0, tokens[:cut], list(range(cut)))])] + [m.step([(0, p, tokens[p:p + 1], [0])]) for p in range(cut, 100)]
            m.release(0)
            return np.concatenate(out)
        base = logits(t)
        for j in (0, 15, 16, 31, 47):
            other = list(t)
            other[j] = (t[j] + 7) % 60
            moved = np.abs(logits(other) - base).max(axis=1)
            assert not moved[:j].any() and not moved[j + window:].any()
            assert (moved[j:j + window] > 1e-5).all()


def test_previous_token_outlives_portions_slots_and_pauses(tmp_path):
    """The pair of tokens an embedding looks at straddles portions; a slot that is used again starts without one."""
    cfg = L.config([L.layer(1, 8, 8, 8, 16, 4)], vocab=50, width=32, bigram=(97, 2147483647, 1000003))
    w = L.random_weights(cfg, 2)
    w["bigram"] = w["bigram"] * 4
    rng = np.random.default_rng(3)
    a, b = rng.integers(0, 50, 9).tolist(), rng.integers(0, 50, 7).tolist()
    wa, wb = L.reference_logits(cfg, w, a), L.reference_logits(cfg, w, b)
    with open_model(tmp_path, cfg, w, f32=True, max_tokens=64, max_seqs=2) as m:
        got_a = [m.step([(0, 0, a[:4], [0, 1, 2, 3])])]
        both = m.step([(1, 0, b[:1], [0]), (0, 4, a[4:6], [0, 1])])
        rest_b = m.step([(1, 1, b[1:], list(range(6)))])  # the other one pauses
        got_a += [both[1:], m.step([(0, 6, a[6:7], [0])]), m.step([(0, 7, a[7:], [0, 1])])]
        assert H.error(np.concatenate(got_a), wa).max() < 3e-5
        assert H.error(np.concatenate([both[:1], rest_b]), wb).max() < 3e-5
        m.release(0)
        assert H.error(m.step([(0, 0, b, list(range(7)))]), wb).max() < 3e-5
        assert H.error(m.step([(0, 0, a, list(range(9)))]), wa).max() < 3e-5  # restarted without a release


def test_each_pass_of_a_loop_has_a_cache_of_its_own(tmp_path):
    """The same layer three times over a wide window, token by token: a pass that read another's rows would be far off."""
    cfg = L.config([L.layer(2, 8, 4, 8, 16, 64, scale=0.5)], vocab=30, width=24, loop=(0, 1, 3))
    w = L.random_weights(cfg, 8)
    t = np.random.default_rng(5).integers(0, 30, 50).tolist()
    want = L.reference_logits(cfg, w, t)
    for f32, tol in ((True, 3e-5), (False, 4e-2)):
        with open_model(tmp_path, cfg, w, f32=f32, max_tokens=64) as m:
            got = np.concatenate([m.step([(0, p, t[p:p + 1], [0])]) for p in range(50)])
        assert H.error(got, want).max() < tol


def test_pages_behind_the_window_serve_other_sequences(tmp_path):
    """A pool that could not hold whole sequences: long ones go on because what leaves the window is given back."""
    cfg = L.config([L.layer(2, 8, 8, 8, 16, 20, experts=2, top=2, ff=8)], vocab=40, width=24, bigram=(11, 3, 5))
    w = L.random_weights(cfg, 6)
    t = np.random.default_rng(2).integers(0, 40, 600).tolist()
    want = L.reference_logits(cfg, w, t)
    with open_model(tmp_path, cfg, w, f32=True, max_tokens=640, max_seqs=3, max_step_tokens=32) as m:
        got = {s: [] for s in range(3)}
        for p in range(0, 600, 10):
            rows = m.step([(s, p, t[p:p + 10], list(range(10))) for s in range(3)])
            for s in range(3):
                got[s].append(rows[s * 10:s * 10 + 10])
        for s in range(3):
            assert H.error(np.concatenate(got[s]), want).max() < 3e-5


def test_designs_share_their_parts(tmp_path):
    """Mixers and feed-forwards of one design in the other: a dense feed-forward beside a mixer, a mixture after one."""
    base = L.config([L.layer(2, 8, 8, 8, 16, 12), L.layer(2, 8, 8, 8, 16, 12, experts=3, top=2, ff=8)], vocab=30, width=24)
    base["layers"][0]["mlp"] = {"kind": "dense", "ff": 20}
    cfg = json.loads(json.dumps(base))
    cfg["layers"][0]["mlp"] = None
    w = L.random_weights(cfg, 1)
    rng = np.random.default_rng(0)
    q = lambda *s: M.from_bf16(M.to_bf16(rng.standard_normal(s) / s[-1] ** 0.5))
    w.update({"l0.norm2": q(24), "l0.mlp.gate": q(20, 24), "l0.mlp.up": q(20, 24), "l0.mlp.down": q(24, 20), "head": q(30, 24)})
    import hybrid_reference as HR
    import latent_moe_reference as R
    t = rng.integers(0, 30, 40).tolist()
    W = {k: v.astype(np.float64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]

    def parallel():
        x = R.embed(t, W, base)
        x = x + R.latent_attention(R.offset_norm(x, W["l0.norm1"], eps), W, "l0.mix.", base["layers"][0]["mixer"], eps) \
            + HR.gated_mlp(R.offset_norm(x, W["l0.norm2"], eps), W, "l0.mlp.")
        x = R.layer(x, W, "l1.", base, 1, eps)
        z = R.offset_norm(x, W["final.norm"], eps) @ W["embed"].T
        return 9.0 * np.tanh(z / 9.0)

    def sequential():
        x = W["embed"][t]
        for i, p in ((0, "l0."), (1, "l1.")):
            x = x + R.latent_attention(HR.rms_norm(x, W[p + "norm1"], eps), W, p + "mix.", base["layers"][i]["mixer"], eps)
            h = HR.rms_norm(x, W[p + "norm2"], eps)
            x = x + (HR.gated_mlp(h, W, p + "mlp.") if i == 0 else R.mixture(h, W, p + "mlp.", base["layers"][1]["mlp"]))
        return HR.rms_norm(x, W["final.norm"], eps) @ W["head"].T

    for arch, want in (("Banevik", parallel()), ("Besudra", sequential())):
        c = dict(base, architecture=arch)
        if arch == "Besudra":
            c.update(logit_softcap=None)
        with open_model(tmp_path / arch, c, w, f32=True, max_tokens=64) as m:
            got = np.concatenate([m.step([(0, 0, t[:30], list(range(30)))])] + [m.step([(0, p, t[p:p + 1], [0])]) for p in range(30, 40)])
        assert H.error(got, want).max() < 3e-5, arch


def test_refusals(tmp_path):
    cfg = L.config([L.layer(2, 8, 8, 8, 16, 12, experts=3, top=2, ff=8)], vocab=30, width=24)
    w = L.random_weights(cfg)

    def refused(change, text, name):
        c = json.loads(json.dumps(cfg))
        change(c)
        with pytest.raises(M.ModelError, match=text):
            open_model(tmp_path / name, c, w)
    refused(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "even", "a")
    refused(lambda c: c["layers"][0]["mlp"]["router"].update(top=4), "out of range", "b")
    refused(lambda c: c["layers"][0]["mlp"].update(kind="other"), "feed-forward kind", "c")
    refused(lambda c: c.update(loop={"start": 1, "stop": 1, "times": 2}), "no layers", "d")
    refused(lambda c: c["layers"][0]["mixer"].update(heads=3), "shape", "e")
