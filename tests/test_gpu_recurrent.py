"""The recurrent kernels (csrc/recurrent.cu) through the C ABI against the plain statements in hybrid_reference.py: ragged
batches, portions that carry state from one call to the next, slots that are used again, odd sizes."""
import ctypes as C

import numpy as np
import pytest

import hybrid_reference as R
from hybrid_step import Step, act_out, dev, lib, plan

pytestmark = pytest.mark.gpu


def run_in_portions(cuts, lens, call):
    """cuts: for every sequence the list of portion lengths. Calls call(step, first tokens) batch by batch until all are through."""
    at = [0] * len(lens)
    k = 0
    while any(a < n for a, n in zip(at, lens)):
        live = [i for i in range(len(lens)) if at[i] < lens[i]]
        part = {i: min(cuts[i][k % len(cuts[i])], lens[i] - at[i]) for i in live}
        call(live, [at[i] for i in live], [part[i] for i in live])
        for i in live:
            at[i] += part[i]
        k += 1


CUTS = {"whole": [[10 ** 9]], "portions": [[2, 17, 1, 40], [33, 3], [5]], "single": [[1]]}


@pytest.mark.parametrize("act", [1, 2])
@pytest.mark.parametrize("cut", CUTS)
@pytest.mark.parametrize("taps,channels", [(4, 200), (2, 64), (3, 130), (1, 24), (7, 40)])
def test_causal_conv(taps, channels, cut, act):
    import torch
    rng = np.random.default_rng(taps)
    lens, slots = [61, 37, 5], [3, 0, 2]
    w, b, ib = rng.standard_normal((channels, taps)), rng.standard_normal(channels), rng.standard_normal(channels)
    ld = channels + 8
    xs = [rng.standard_normal((n, channels)) for n in lens]
    want = [R.silu(R.causal_conv(x + ib, w, b)) for x in xs]
    got = [np.zeros((n, channels)) for n in lens]
    state = torch.full((4, max(taps - 1, 1), channels), float("nan"), device="cuda")  # a fresh sequence must not read its slot
    wd, bd, ibd = dev(w), dev(b), dev(ib)
    cuts = (CUTS[cut] * 3)[:3]

    def call(live, pos0, part):
        st = Step(part, pos0, [slots[i] for i in live])
        rows = np.zeros((st.n_tok, ld))
        rows[:, :channels] = np.concatenate([xs[i][p:p + n] for i, p, n in zip(live, pos0, part)])
        x = dev(rows)
        out, hi, lo = (torch.zeros(st.n_tok, channels, device="cuda", dtype=t) for t in (torch.float32, torch.bfloat16, torch.bfloat16))
        o = act_out(out, hi, lo)
        lib(lib().ingot_causal_conv(C.byref(st.c), x.data_ptr(), ld, ibd.data_ptr(), wd.data_ptr(), bd.data_ptr(), taps, channels, act,
                                    state.data_ptr(), C.byref(o), None))
        torch.cuda.synchronize()
        assert torch.equal(hi, out.bfloat16()) and torch.equal(lo, (out - hi.float()).bfloat16())
        r = 0
        for i, p, n in zip(live, pos0, part):
            got[i][p:p + n] = out[r:r + n].cpu().numpy()
            r += n

    run_in_portions(cuts, lens, call)
    for g, e in zip(got, want):
        assert np.abs(g - e).max() < 2e-5


@pytest.mark.parametrize("exact", [0, 1])
@pytest.mark.parametrize("cut", CUTS)
@pytest.mark.parametrize("inner,n_state", [(96, 16), (40, 20), (8, 1), (72, 33), (24, 70), (36, 5)])
def test_selective_scan(inner, n_state, cut, exact):
    import torch
    rng = np.random.default_rng(inner + n_state)
    lens, slots = [101, 64, 7], [1, 3, 0]
    pad = lib().ingot_scan_state_pad(n_state)
    assert pad >= n_state and pad % 8 == 0
    A = -np.exp(rng.uniform(-1, 2, (inner, n_state)))
    D, bias = rng.standard_normal(inner), rng.uniform(-4, -1, inner)
    x, raw, z = ([rng.standard_normal((n, inner)) for n in lens] for _ in range(3))
    B, Cm = ([rng.standard_normal((n, n_state)) for n in lens] for _ in range(2))
    want = [R.selective_scan(x[i], R.softplus(raw[i] + bias), A, B[i], Cm[i], D) * R.silu(z[i]) for i in range(3)]
    got = [np.zeros((n, inner)) for n in lens]
    a2 = np.zeros((inner, pad))
    a2[:, :n_state] = A * np.log2(np.e)
    a2d, dd, bd = dev(a2), dev(D), dev(bias)
    state = torch.full((4, inner, pad), float("nan"), device="cuda")
    cuts = (CUTS[cut] * 3)[:3]

    def call(live, pos0, part):
        st = Step(part, pos0, [slots[i] for i in live])
        take = lambda a: np.concatenate([a[i][p:p + n] for i, p, n in zip(live, pos0, part)])
        bc = np.zeros((st.n_tok, 4 + 2 * pad))
        bc[:, 4:4 + n_state] = take(B)
        bc[:, 4 + pad:4 + pad + n_state] = take(Cm)
        xz = np.concatenate([take(x), take(z)], axis=1)
        xd, td, bcd = dev(xz), dev(take(raw)), dev(bc)
        out = torch.zeros(st.n_tok, inner, device="cuda")
        o = act_out(out)
        pl = plan(part, 16, inner * (pad + 1))
        lib(lib().ingot_selective_scan(C.byref(st.c), C.byref(pl.c), xd.data_ptr(), 2 * inner, td.data_ptr(), inner, bd.data_ptr(),
                                       bcd.data_ptr(), 4 + 2 * pad, 4, 4 + pad, xd.data_ptr() + 4 * inner, 2 * inner, a2d.data_ptr(),
                                       dd.data_ptr(), state.data_ptr(), inner, n_state, exact, C.byref(o), None))
        torch.cuda.synchronize()
        r = 0
        for i, p, n in zip(live, pos0, part):
            got[i][p:p + n] = out[r:r + n].cpu().numpy()
            r += n

    run_in_portions(cuts, lens, call)
    for g, e in zip(got, want):
        assert np.abs(g - e).max() < 3e-5 * max(1.0, np.abs(e).max())


@pytest.mark.parametrize("exact", [0, 1])
@pytest.mark.parametrize("cut", CUTS)
@pytest.mark.parametrize("width,block", [(96, 24), (200, 200), (24, 8)])
def test_gated_lru(width, block, cut, exact):
    import torch
    rng = np.random.default_rng(width)
    lens, slots = [90, 33, 4], [2, 1, 3]
    br, bi, yb = (rng.standard_normal(width) for _ in range(3))
    lam = rng.uniform(-6, 1, width)  # from nearly no decay to a fast one
    u, gr, gi, y = ([rng.standard_normal((n, width)) for n in lens] for _ in range(4))
    want = [0.75 * R.gated_lru_scan(u[i], R.sigmoid(gr[i] + br), R.sigmoid(gi[i] + bi), lam) * R.gelu_tanh(y[i] + yb) for i in range(3)]
    got = [np.zeros((n, width)) for n in lens]
    dv = [dev(v) for v in (br, bi, R.softplus(lam), yb)]
    state = torch.full((4, width), float("nan"), device="cuda")
    cuts = (CUTS[cut] * 3)[:3]

    def call(live, pos0, part):
        st = Step(part, pos0, [slots[i] for i in live])
        take = lambda a: np.concatenate([a[i][p:p + n] for i, p, n in zip(live, pos0, part)])
        g = np.stack([take(gr).reshape(st.n_tok, -1, block), take(gi).reshape(st.n_tok, -1, block)], axis=2).reshape(st.n_tok, 2 * width)
        ud, gd, yd = dev(take(u)), dev(g), dev(take(y))
        out = torch.zeros(st.n_tok, width, device="cuda")
        o = act_out(out)
        pl = plan(part, 16, 2 * width)
        lib(lib().ingot_gated_lru(C.byref(st.c), C.byref(pl.c), ud.data_ptr(), width, gd.data_ptr(), 2 * width, block, dv[0].data_ptr(),
                                  dv[1].data_ptr(), dv[2].data_ptr(), yd.data_ptr(), width, dv[3].data_ptr(), state.data_ptr(), width, 0.75,
                                  exact, C.byref(o), None))
        torch.cuda.synchronize()
        r = 0
        for i, p, n in zip(live, pos0, part):
            got[i][p:p + n] = out[r:r + n].cpu().numpy()
            r += n

    run_in_portions(cuts, lens, call)
    for g, e in zip(got, want):
        assert np.abs(g - e).max() < 2e-5


def test_long_memory_does_not_drift():
    """A channel that hardly decays, fed one token at a time: the exact forms stay within rounding of float64."""
    import torch
    n, inner, pad = 600, 8, 8
    rng = np.random.default_rng(1)
    A = -np.full((inner, 1), 1e-3)
    x, raw, z = rng.standard_normal((n, inner)) + 1, np.zeros((n, inner)), np.ones((n, inner))
    ones = np.ones((n, 1))
    want = R.selective_scan(x, R.softplus(raw), A, ones, ones, np.zeros(inner)) * R.silu(z)
    a2 = np.zeros((inner, pad))
    a2[:, :1] = A * np.log2(np.e)
    a2d, zero = dev(a2), dev(np.zeros(inner))
    state = torch.zeros(1, inner, pad, device="cuda")
    bc = np.zeros((1, 2 * pad))
    bc[0, 0] = bc[0, pad] = 1
    bcd = dev(bc)
    got = np.zeros((n, inner))
    for t in range(n):
        st = Step([1], [t], [0])
        xd, td, zd = dev(x[t:t + 1]), dev(raw[t:t + 1]), dev(z[t:t + 1])
        out = torch.zeros(1, inner, device="cuda")
        o = act_out(out)
        pl = plan([1], 16, inner * (pad + 1))
        lib(lib().ingot_selective_scan(C.byref(st.c), C.byref(pl.c), xd.data_ptr(), inner, td.data_ptr(), inner, zero.data_ptr(), bcd.data_ptr(),
                                       2 * pad, 0, pad, zd.data_ptr(), inner, a2d.data_ptr(), zero.data_ptr(), state.data_ptr(), inner, 1, 1,
                                       C.byref(o), None))
        got[t] = out.cpu().numpy()
    assert (np.abs(got - want) / np.abs(want).max()).max() < 1e-6
