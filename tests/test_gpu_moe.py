"""Mixture of experts: routing and the plain products (csrc/moe.cu), the grouped tcgen05 product (backend/linear_sm100.cu)."""
import ctypes as C

import numpy as np
import pytest

import latent_moe_reference as R
from hybrid_step import dev, lib
from ingot_b200 import models as M

pytestmark = pytest.mark.gpu


def route(z, n_expert, top):
    import torch
    n = z.shape[0]
    zd = dev(z)
    i = lambda k: torch.full((k,), -7, device="cuda", dtype=torch.int32)
    f = lambda k: torch.zeros(k, device="cuda")
    expert, weight, start, row, pair, row_w = i(n * top), f(n * top), i(n_expert + 1), i(n * top), i(n * top), f(n * top)
    lib(lib().ingot_moe_route(zd.data_ptr(), z.shape[1], n, n_expert, top, *[t.data_ptr() for t in (expert, weight, start, row, pair, row_w)], None))
    torch.cuda.synchronize()
    return [t.cpu().numpy() for t in (expert, weight, start, row, pair, row_w)]


@pytest.mark.parametrize("n,experts,top", [(1, 5, 2), (7, 12, 1), (64, 3, 3), (300, 64, 6), (1000, 40, 5), (5, 300, 8), (2049, 8, 2), (33, 1, 1)])
def test_routing(n, experts, top):
    rng = np.random.default_rng(n)
    z = np.zeros((n, experts + 3), np.float32)
    z[:, :experts] = rng.standard_normal((n, experts)) * 3
    z[:, experts:] = 1e9  # padding columns are not experts
    expert, weight, start, row, pair, row_w = route(z, experts, top)
    best, s = R.route(z[:, :experts].astype(np.float64), np.eye(experts), top)
    assert np.array_equal(expert.reshape(n, top), best) and np.abs(weight.reshape(n, top) - s).max() < 1e-6
    order = np.argsort(expert, kind="stable")
    assert np.array_equal(pair, order) and np.array_equal(row[order], np.arange(n * top)) and np.array_equal(row_w, weight[order])
    assert np.array_equal(start, np.searchsorted(np.sort(expert), np.arange(experts + 1)))


def test_routing_of_ties_and_values_that_are_not_numbers():
    z = np.array([[1, 2, 2, 1], [np.nan] * 4, [np.nan, 0, np.nan, -5], [-np.inf] * 4], np.float32)
    expert = route(z, 4, 3)[0].reshape(4, 3)
    assert expert.tolist() == [[1, 2, 0], [0, 1, 2], [1, 3, 0], [0, 1, 2]]


class CGrouped(C.Structure):
    _fields_ = [("a_hi", C.c_void_p), ("a_lo", C.c_void_p), ("n_rows", C.c_int), ("rows_per_group", C.c_int), ("w", C.c_void_p), ("n_in", C.c_int),
                ("n_out", C.c_int), ("n_groups", C.c_int), ("group_start", C.c_void_p), ("row_scale", C.c_void_p), ("act", C.c_int), ("out", C.c_void_p),
                ("out_hi", C.c_void_p), ("out_lo", C.c_void_p)]


def bf16(x):
    import torch
    return torch.from_numpy(np.ascontiguousarray(x, dtype=np.float32)).cuda().bfloat16()


CASES = [([5], 16, 24), ([3, 0, 1, 7], 72, 40), ([200, 128, 0, 1, 129], 136, 264), ([0, 0, 900, 30], 256, 512), ([1] * 40 + [0] * 10, 64, 128), ([40] * 70, 128, 96)]


@pytest.mark.parametrize("planes", [1, 2])
@pytest.mark.parametrize("counts,n_in,n_out", CASES, ids=str)
def test_grouped_product(counts, n_in, n_out, planes):
    """f32 results, and the activation folded in with bf16 results; groups that are empty, shorter and longer than a tile."""
    import torch
    L = M.lib()
    L.ingot_linear_ws_create_bf16.argtypes = [C.POINTER(C.c_void_p), C.c_int, C.c_int, C.c_int]
    L.ingot_linear_ws_status.argtypes = L.ingot_linear_ws_destroy.argtypes = [C.c_void_p]
    L.ingot_grouped_tc_run.argtypes = [C.c_void_p, C.c_void_p, C.c_void_p]
    rng = np.random.default_rng(n_in)
    rows, groups = sum(counts), len(counts)
    x, w = rng.standard_normal((rows, n_in)), rng.standard_normal((groups, n_out, n_in)) / n_in ** 0.5
    start = np.concatenate([[0], np.cumsum(counts)])
    hi = bf16(x)
    lo = bf16(x - hi.float().cpu().numpy())
    wd, sd = bf16(w), dev(start, np.int32)
    scale = rng.random(rows) + 0.2
    sc = dev(scale)
    seen = hi.double() + (lo.double() if planes > 1 else 0)
    want = torch.cat([seen[a:b] @ wd[g].double().T for g, (a, b) in enumerate(zip(start[:-1], start[1:]))]).cpu().numpy()
    ws = C.c_void_p()
    assert L.ingot_linear_ws_create_bf16(C.byref(ws), 8, 8, 8) == 0
    try:
        out = torch.full((rows, n_out), np.nan, device="cuda")
        g = CGrouped(hi.data_ptr(), lo.data_ptr() if planes > 1 else None, rows, max(counts), wd.data_ptr(), n_in, n_out, groups, sd.data_ptr(), None, 0,
                     out.data_ptr(), None, None)
        assert L.ingot_grouped_tc_run(ws, C.byref(g), None) == 0
        torch.cuda.synchronize()
        assert L.ingot_linear_ws_status(ws) == 0
        assert np.abs(out.cpu().numpy() - want).max() < 2e-5
        o_hi, o_lo = (torch.full((rows, n_out), np.nan, device="cuda", dtype=torch.bfloat16) for _ in range(2))
        g.row_scale, g.act, g.out, g.out_hi, g.out_lo = sc.data_ptr(), 1, None, o_hi.data_ptr(), o_lo.data_ptr()
        assert L.ingot_grouped_tc_run(ws, C.byref(g), None) == 0
        torch.cuda.synchronize()
        act = np.square(np.maximum(want * scale[:, None], 0))
        assert np.abs((o_hi.double() + o_lo.double()).cpu().numpy() - act).max() < 1e-4 * max(1, act.max())
    finally:
        L.ingot_linear_ws_destroy(ws)


@pytest.mark.parametrize("n,experts,top,d,ff", [(1, 4, 2, 40, 24), (9, 5, 5, 64, 16), (130, 12, 3, 48, 72), (600, 3, 1, 16, 8)])
def test_plain_experts_against_the_mixture(n, experts, top, d, ff):
    """Routing, both products and the sum into the residual, against the plain mixture."""
    import torch
    rng = np.random.default_rng(d)
    W = {"router": rng.standard_normal((experts, d)) / d ** 0.5}
    up = bf16(rng.standard_normal((experts, ff, d)) / d ** 0.5)
    down = bf16(rng.standard_normal((experts, d, ff)) / ff ** 0.5)
    for e in range(experts):
        W[f"e{e}.up"], W[f"e{e}.down"] = up[e].double().cpu().numpy(), down[e].double().cpu().numpy()
    h, x = rng.standard_normal((n, d)).astype(np.float32), rng.standard_normal((n, d)).astype(np.float32)
    want = x + R.mixture(h.astype(np.float64), W, "", {"router": {"top": top}})
    _, _, start, row, pair, row_w = route((h.astype(np.float64) @ W["router"].T).astype(np.float32), experts, top)
    hd, xd, sd, rd, pd, wd = dev(h), dev(x), dev(start, np.int32), dev(row, np.int32), dev(pair, np.int32), dev(row_w)
    mid, out = torch.zeros(n * top, ff, device="cuda"), torch.zeros(n * top, d, device="cuda")
    p = lambda t: t.data_ptr()
    lib(lib().ingot_moe_linear(p(mid), p(up), p(hd), d, d, ff, experts, n * top, p(sd), p(pd), top, p(wd), 1, None))
    lib(lib().ingot_moe_linear(p(out), p(down), p(mid), ff, ff, d, experts, n * top, p(sd), None, top, None, 0, None))
    lib(lib().ingot_moe_add(p(xd), p(out), p(rd), n, top, d, None))
    torch.cuda.synchronize()
    assert np.abs(xd.cpu().numpy() - want).max() < 1e-4
    planes = bf16(h)
    gathered = torch.zeros(n * top, d, device="cuda", dtype=torch.bfloat16)
    lib(lib().ingot_moe_gather(p(gathered), None, p(planes), None, p(pd), n * top, None, top, d, None))
    torch.cuda.synchronize()
    assert torch.equal(gathered, planes[torch.from_numpy(pair // top).cuda().long()])
