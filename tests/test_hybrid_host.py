"""Host side of the model-folder backends without a GPU, and the plain implementation checked against itself."""
import os
import shutil
import subprocess

import numpy as np
import pytest

import hybrid_models as H
import hybrid_reference as R

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BACKEND = os.path.join(ROOT, "inference-agent_b200", "backend")


def test_host_units(tmp_path):
    cxx = shutil.which("g++")
    if not cxx:
        pytest.skip("no g++")
    cfg = H.config([H.mamba(12, 3, 2, 3)], vocab=11, width=10)
    good = H.write(tmp_path / "good", cfg, H.random_weights(cfg))
    bad = H.write(tmp_path / "bad", cfg, H.random_weights(cfg))
    with open(os.path.join(bad, "model.safetensors"), "r+b") as f:
        f.truncate(os.path.getsize(f.name) - 6)
    exe = str(tmp_path / "host_units")
    subprocess.run([cxx, "-std=c++20", "-O1", "-Wall", "-Wextra", "-Werror", "-fsanitize=address,undefined", "-I", BACKEND,
                    os.path.join(ROOT, "tests", "native", "host_units.cpp"), os.path.join(BACKEND, "model_dir.cpp"), "-o", exe], check=True, timeout=300)
    r = subprocess.run([exe, good, bad], capture_output=True, text=True, timeout=120)
    assert r.returncode == 0 and r.stdout == "ok\n", r.stdout + r.stderr


def test_bf16_rounding_is_to_nearest_even():
    from ingot_b200.models import from_bf16, to_bf16
    x = np.array([1.0, 1 + 2 ** -8, 1 + 3 * 2 ** -8, -1.00390625 * 1.001, 3e38], dtype=np.float32)
    assert from_bf16(to_bf16(x))[:3].tolist() == [1.0, 1.0, 1 + 2 ** -6]
    assert abs(from_bf16(to_bf16(x))[3] / x[3] - 1) < 2 ** -8


def test_plain_mechanisms():
    rng = np.random.default_rng(0)
    vis = R.chunk_visible(9, 4)
    assert vis[3].nonzero()[0].tolist() == [0, 1, 2, 3] and vis[4].nonzero()[0].tolist() == [4] and vis[8].nonzero()[0].tolist() == [8]
    x, w, b = rng.standard_normal((7, 3)), rng.standard_normal((3, 4)), rng.standard_normal(3)
    y = R.causal_conv(x, w, b)
    assert np.allclose(y[0], b + w[:, 3] * x[0]) and np.allclose(y[5], b + sum(w[:, j] * x[2 + j] for j in range(4)))
    # a scan cut in two with its state handed over is the scan
    lam, r, i, u = rng.standard_normal(3), rng.random((7, 3)), rng.random((7, 3)), rng.standard_normal((7, 3))
    whole = R.gated_lru_scan(u, r, i, lam)
    assert np.allclose(R.gated_lru_scan(u[4:], r[4:], i[4:], lam, whole[3]), whole[4:])
    # scan of one step: S = dt x B, y = S C + D x
    A, dt, B, C, D = -rng.random((3, 2)), rng.random((1, 3)), rng.standard_normal((1, 2)), rng.standard_normal((1, 2)), rng.standard_normal(3)
    got = R.selective_scan(x[:1], dt, A, B, C, D)
    assert np.allclose(got[0], dt[0] * x[0] * (B[0] @ C[0]) + D * x[0])
    # the model is causal: later tokens do not change earlier logits
    cfg = H.config([H.mamba(12, 3, 2, 3), H.parallel(4, 2, 6, 5, 8, 2, 2, ff=9)], vocab=13, width=10)
    wts = H.random_weights(cfg)
    t = rng.integers(0, 13, 17).tolist()
    assert np.allclose(H.reference_logits(cfg, wts, t)[:9], H.reference_logits(cfg, wts, t[:9]))
