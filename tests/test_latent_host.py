"""The plain implementation of the latent / mixture design checked against itself, without a GPU."""
import numpy as np

import latent_moe_models as L
import latent_moe_reference as R


def test_window_and_sink():
    see = R.window_visible(9, 3)
    assert see[5].nonzero()[0].tolist() == [3, 4, 5] and see[0].nonzero()[0].tolist() == [0]
    assert R.window_visible(6, 0)[5].all() and R.window_visible(4, 1).sum() == 4
    p = R.softmax_with_sink(np.array([[0.0, -np.inf, np.log(2.0)]]), np.log(5.0))
    assert np.allclose(p, [[1 / 8, 0, 2 / 8]])


def test_rotation_depends_on_the_distance_only():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal(10), rng.standard_normal(10)
    at = lambda v, p: R.rotate(v[None], [p], 8, 100.0)[0]
    assert np.allclose(at(q, 7) @ at(k, 3), at(q, 1007) @ at(k, 1003)) and not np.allclose(at(q, 7) @ at(k, 3), at(q, 8) @ at(k, 3))
    assert np.allclose(at(q, 0), q) and np.allclose(at(q, 5)[8:], q[8:])
    one = at(np.eye(10)[1], 3)  # value 1 turns towards value 5
    assert np.allclose(one[[1, 5]], [np.cos(3 * 100 ** -0.25), np.sin(3 * 100 ** -0.25)])


def test_bigram_rows():
    assert R.bigram_rows([4, 9, 9], 10, 3, 7).tolist() == [10, (12 + 63) % 10, (27 + 63) % 10]


def test_routing_takes_the_largest_and_keeps_their_scores():
    h, w = np.array([[1.0, 0.0]]), np.array([[0.1, 5], [2.0, 5], [-1.0, 5], [1.0, 5]])
    best, s = R.route(h, w, 2)
    assert best.tolist() == [[1, 3]] and np.allclose(s, 1 / (1 + np.exp([[-2.0, -1.0]])))


def test_latent_attention_on_the_rows_is_attention_on_the_expansion():
    """Taking the query into the latent space and the values out of it afterwards gives the same result."""
    rng = np.random.default_rng(1)
    H, k, r, v, c, n = 3, 4, 2, 5, 6, 11
    m = {"heads": H, "dim": k, "rot_dim": r, "vdim": v, "kv_rank": c, "scale": 0.3, "rot": {"base": 50.0, "dims": r}, "mask": {"size": 4}}
    W = {"q": rng.standard_normal((H * (k + r), 8)), "dkv": rng.standard_normal((c + r, 8)), "dkv.norm": rng.standard_normal(c), "uk": rng.standard_normal((H * k, c)),
         "uv": rng.standard_normal((H * v, c)), "sink": rng.standard_normal(H), "o": np.eye(H * v)}
    h = rng.standard_normal((n, 8))
    want = R.latent_attention(h, W, "", m, 1e-5)
    lat, kr = R.latent(h, W, "", m, 1e-5)
    q = (h @ W["q"].T).reshape(n, H, k + r)
    for i in range(H):
        rows = np.concatenate([q[:, i, :k] @ W["uk"][i * k:(i + 1) * k], R.rotate(q[:, i, k:], range(n), r, 50.0)], axis=1)
        s = np.where(R.window_visible(n, 4), rows @ np.concatenate([lat, kr], axis=1).T * 0.3, -np.inf)
        assert np.allclose(R.softmax_with_sink(s, W["sink"][i]) @ lat @ W["uv"][i * v:(i + 1) * v].T, want[:, i * v:(i + 1) * v])


def test_loop_order_and_causality():
    cfg = L.config([L.layer(2, 4, 2, 4, 6, 5, experts=3, top=2, ff=8) for _ in range(4)], vocab=20, width=12, loop=(1, 3, 2), bigram=(11, 5, 3))
    assert [i for i, _ in R.layer_runs(cfg)] == [0, 1, 2, 1, 2, 3] and [e for _, e in R.layer_runs(cfg)] == [False, True, False, True, False, False]
    w = L.random_weights(cfg)
    t = np.random.default_rng(0).integers(0, 20, 17).tolist()
    assert np.allclose(L.reference_logits(cfg, w, t)[:9], L.reference_logits(cfg, w, t[:9]))
    assert np.abs(L.reference_logits(cfg, w, t)).max() < 9.0
