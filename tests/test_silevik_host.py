"""The plain implementation of the sandwich-normed design checked against itself, without a GPU."""
import numpy as np

import hybrid_models as H
import silevik_models as S
import silevik_reference as R


def test_norms():
    x = np.array([[1.0, 3.0, 5.0, 7.0]])
    n = R.layer_norm(x, 2.0, 1.0, 0.0)
    assert np.allclose((n - 1) / 2, (x - 4) / np.sqrt(5)) and np.allclose(R.layer_norm(x + 100, 2.0, 1.0, 0.0), n)
    assert np.allclose(R.rms_norm(x, 1.0, 0.0), x / np.sqrt(21))


def test_rotation_turns_neighbours_and_depends_on_the_distance_only():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))
    at = lambda v, p: R.rotate(v, [p], 8, 100.0)[0, 0]
    assert np.allclose(at(q, 7) @ at(k, 3), at(q, 1007) @ at(k, 1003)) and not np.allclose(at(q, 7) @ at(k, 3), at(q, 8) @ at(k, 3))
    assert np.allclose(at(q, 5)[8:], q[0, 0, 8:])
    one = at(np.eye(10)[2][None, None], 3)  # value 2 turns towards value 3
    assert np.allclose(one[[2, 3]], [np.cos(3 * 100 ** -0.25), np.sin(3 * 100 ** -0.25)])


def test_scaled_frequencies():
    """Pairs that turn often keep their frequency, those that turn rarely are slowed by the factor, with a ramp over the index between."""
    plain, one = R.frequencies(32, 10000.0)
    f, gain = R.frequencies(32, 10000.0, {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0})
    ratio = plain / f
    assert one == 1.0 and np.isclose(gain, 0.1 * np.log(8) + 1)
    assert np.allclose(ratio[:5], 1) and np.allclose(ratio[-4:], 8) and (np.diff(ratio) >= -1e-12).all()
    turns = 4096 * plain / (2 * np.pi)
    assert (turns[np.isclose(ratio, 1)] > 16).all() and (turns[np.isclose(ratio, 8)] < 1.5).all()


def test_window_and_sink():
    assert R.visible(9, 3)[5].nonzero()[0].tolist() == [3, 4, 5] and R.visible(6, 0)[5].all() and R.visible(4, 1).sum() == 4
    assert np.allclose(R.softmax(np.array([[0.0, -np.inf, np.log(2.0)]]), np.log(5.0)), [[1 / 8, 0, 2 / 8]])
    assert np.allclose(R.softmax(np.array([[0.0, np.log(3.0)]])), [[1 / 4, 3 / 4]])


def test_routing_by_groups():
    w = np.eye(6)
    h = np.log(np.array([[0.4, 0.1, 0.3, 0.05, 0.1, 0.05]]))
    zero = np.zeros(6)
    assert R.route(h, w, zero, 3, 1, 1, 1.0)[0].tolist() == [[0, 2, 1]]
    assert R.route(h, w, zero, 2, 3, 1, 1.0)[0].tolist() == [[0, 1]]        # the best pair holds the best output
    chosen, weight = R.route(h, w, np.array([-9, -9, -9, -9, -1, -2.0]), 3, 3, 2, 2.0)
    assert chosen.tolist() == [[4, 5, 0]]                                     # corrections choose
    assert np.allclose(weight, 2 * np.array([[0.1, 0.05, 0.4]]) / 0.55)       # and do not weigh


def test_identity_and_shared_experts():
    rng = np.random.default_rng(1)
    W = {"router": rng.standard_normal((3, 4)), "correction": np.array([-9, -9, 9.0]), "shared.sg": np.zeros((1, 4))}
    for e in ("e0", "e1", "shared"):
        W.update({f"{e}.gate": rng.standard_normal((5, 4)), f"{e}.up": rng.standard_normal((5, 4)), f"{e}.down": rng.standard_normal((4, 5))})
    h = rng.standard_normal((2, 4))
    mlp = {"router": {"experts": 2, "identity": 1, "top": 1, "scale": 3.0, "groups": None}, "shared": {"ff": 5}}
    assert np.allclose(R.mixture(h, W, "", mlp), 3 * h + 0.5 * R.gated_mlp(h, W, "shared."))


def test_causality_and_value_mixing():
    cfg = S.config([S.layer("attention", 4, 2, 8, 6, 5, rot=4, mlp=S.moe(3, 1, 2, (2, 1), 8, 6)), S.layer("attention_3", 2, 2, 8, 6, rot=8, scaling=(2.0, 16, 4.0, 1.0), mlp=S.dense(9)),
                    S.layer("attention_2", 2, 2, 4, 6)], vocab=20, width=12)
    w = S.random_weights(cfg)
    t = np.random.default_rng(0).integers(0, 20, 17).tolist()
    full = S.reference_logits(cfg, w, t)
    assert np.allclose(full[:9], S.reference_logits(cfg, w, t[:9]))
    w2 = dict(w)
    w2["l0.mix.vmix"] = w["l0.mix.vmix"] * 0
    assert np.array_equal(S.reference_logits(cfg, w2, t), full)  # the first one's is not used
    w2["l2.mix.vmix"] = w["l2.mix.vmix"] * 0
    assert H.error(S.reference_logits(cfg, w2, t), full).max() > 1e-3
