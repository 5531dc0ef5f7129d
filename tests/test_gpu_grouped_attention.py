"""Grouped-query attention over joined rows (csrc/attn_gqa.cu, attn_gqa_sm100.cu) through the C ABI against silevik_reference.py: both cache
types, every kernel, lengths that need padding, norms, rotations, mixed values, sinks and gates, pages in random order that leave with the
window, single keys that stand out at every edge."""
import ctypes as C

import numpy as np
import pytest

import silevik_reference as R
from hybrid_step import Step, act_out, dev, lib

pytestmark = pytest.mark.gpu
F32, F16 = 0, 1
EPS = 1e-5
NORMS = {None: 0, "head": 1, "whole": 2}


class CShape(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("n_head", "n_head_kv", "dim", "vdim", "dim_count", "rot_dims", "norm")]


class Shape:
    def __init__(self, heads, kv_heads, dim, vdim, window=0, rot=0, base=300.0, scaling=None, norm=None, gate=None, sink=False, mix=None, scale=None):
        self.heads, self.kv, self.dim, self.vdim, self.window, self.rot, self.norm, self.gate, self.sink, self.mix = heads, kv_heads, dim, vdim, window, rot, norm, gate, sink, mix
        up = lambda v: (v + 15) // 16 * 16
        self.dim_p, self.vdim_p = up(dim), up(vdim)
        self.c = CShape(heads, kv_heads, self.dim_p, self.vdim_p, dim, rot, NORMS[norm])
        self.scale = 1.3 / dim ** 0.5 if scale is None else scale
        self.base, self.scaling = base, scaling

    def parts(self):
        """(heads, size, padded) of the columns of a projection row."""
        out = [(self.heads, self.dim, self.dim_p), (self.kv, self.dim, self.dim_p), (self.kv, self.vdim, self.vdim_p)]
        if self.gate:
            out.append((self.heads, self.vdim, self.vdim_p) if self.gate == "element" else (1, self.heads, (self.heads + 7) // 8 * 8))
        return out


class Weights:
    def __init__(self, s, seed=0, gain=1.0):
        rng = np.random.default_rng(seed)
        n = {None: (0, 0), "head": (s.dim, s.dim), "whole": (s.heads * s.dim, s.kv * s.dim)}[s.norm]
        self.q, self.k = (gain * (1 + 0.3 * rng.standard_normal(m)) for m in n)
        self.sink = rng.standard_normal(s.heads) + 1.0 if s.sink else None


def sequence(s, n, rng):
    """Random q, k, v (and gate logits), and the first mixing layer's values."""
    x = [rng.standard_normal((n, h, d)) for h, d, _ in s.parts()]
    return x + [rng.standard_normal((n, s.kv, s.vdim))]


def reference(s, x, w):
    n, (q, k, v), first = x[0].shape[0], x[:3], x[-1]
    if s.norm == "whole":
        q, k = (R.rms_norm(a.reshape(n, -1), b, EPS).reshape(a.shape) for a, b in ((q, w.q), (k, w.k)))
    elif s.norm == "head":
        q, k = R.rms_norm(q, w.q, EPS), R.rms_norm(k, w.k, EPS)
    if s.rot:
        q, k = (R.rotate(a, range(n), s.rot, s.base, s.scaling) for a in (q, k))
    if s.mix is not None:
        v = R.mix_values(v, first, s.mix)
    y = R.attend(q, k, v, s.scale, s.window, w.sink)
    if s.gate:
        y = y * (R.sigmoid(x[3]) if s.gate == "element" else R.sigmoid(x[3]).reshape(n, s.heads, 1))
    return y


def pad(x, padded):
    n, h, d = x.shape
    out = np.zeros((n, h, padded))
    out[:, :, :d] = x
    return out.reshape(n, -1)


def run(s, seqs, cuts, w, dtype, impl, seed=0):
    """cuts: portion lengths per sequence (repeated). Pages behind the window are not in the tables. impl: per portion as the library
    chooses (0), or the kernel named. Returns [n, heads, vdim] per sequence."""
    import torch
    rng = np.random.default_rng(seed)
    pages = [(x[0].shape[0] + 15) // 16 for x in seqs]
    order = rng.permutation(sum(pages) + 3).astype(np.int32)
    tables = np.split(order[:sum(pages)], np.cumsum(pages)[:-1])
    h = C.c_void_p()
    lib(lib().ingot_skv_create_joined(C.byref(h), 2, s.kv, s.dim_p + s.vdim_p, dtype, s.window, len(order)))
    f, gain = R.frequencies(s.rot, s.base, s.scaling) if s.rot else (np.zeros(1), 1.0)
    turns = dev(f / (2 * np.pi), np.float64)
    qn, kn = (None if s.norm is None else dev(pad(a.reshape(1, -1, s.dim), s.dim_p)) for a in (w.q, w.k))
    sink = None if w.sink is None else dev(w.sink)
    p = lambda t: None if t is None else t.data_ptr()
    off = np.cumsum([0] + [h_ * d for h_, _, d in s.parts()]).tolist()
    outs = [np.zeros((x[0].shape[0], s.heads, s.vdim)) for x in seqs]
    done, k = [0] * len(seqs), 0
    try:
        while any(d < x[0].shape[0] for d, x in zip(done, seqs)):
            live = [i for i, x in enumerate(seqs) if done[i] < x[0].shape[0]]
            part = [min(cuts[i][k % len(cuts[i])], seqs[i][0].shape[0] - done[i]) for i in live]
            st = Step(part, [done[i] for i in live], [0] * len(live))
            n_tok = st.n_tok
            rows = lambda j: np.concatenate([seqs[i][j][done[i]:done[i] + n] for i, n in zip(live, part)])
            proj = dev(np.concatenate([pad(rows(j), d) for j, (_, _, d) in enumerate(s.parts())], axis=1))
            first_values = dev(pad(rows(-1), s.vdim_p))
            first = [max(0, done[i] - s.window + 1) // 16 if s.window else 0 for i in live]
            width = max((done[i] + n + 15) // 16 - f0 for i, n, f0 in zip(live, part, first))
            tab = np.full((len(live), width), -1, np.int32)
            for r, (i, n, f0) in enumerate(zip(live, part, first)):
                tab[r, :(done[i] + n + 15) // 16 - f0] = tables[i][f0:(done[i] + n + 15) // 16]
            td, fd = dev(tab, np.int32), dev(first, np.int32)
            q = torch.zeros(n_tok, s.heads, s.dim_p, device="cuda", dtype=torch.float32 if dtype == F32 else torch.float16)
            out = torch.zeros(n_tok, s.heads * s.vdim_p, device="cuda")
            hi, lo = (torch.zeros(n_tok, s.heads * s.vdim_p, device="cuda", dtype=torch.bfloat16) for _ in range(2))
            oo = act_out(out, hi, lo)
            for layer in (1, 0):
                lib(lib().ingot_gqa_append(h, layer, C.byref(st.c), p(proj), proj.shape[1], off[0], off[1], off[2], C.byref(s.c), p(qn), p(kn), EPS, p(turns), gain,
                                           p(first_values) if s.mix is not None else None, 0, 0.0 if s.mix is None else s.mix, p(q), p(td), p(fd), width, None))
            lib(lib().ingot_gqa_attend(h, 0, C.byref(st.c), p(q), C.byref(s.c), s.scale, p(sink), proj.data_ptr() + 4 * off[3] if s.gate else None, proj.shape[1],
                                       int(s.gate == "head"), C.byref(oo), p(td), p(fd), width, impl, None))
            torch.cuda.synchronize()
            status = C.c_int(-1)
            lib(lib().ingot_skv_status(h, None, C.byref(status)))
            assert status.value == 0
            assert ((hi.float() + lo.float() - out).abs().max() <= 1e-4 * out.abs().max()).item()  # the bf16 pair is the f32 result
            res = out.cpu().numpy().reshape(n_tok, s.heads, s.vdim_p)
            assert not res[:, :, s.vdim:].any()
            r = 0
            for i, n in zip(live, part):
                outs[i][done[i]:done[i] + n] = res[r:r + n, :, :s.vdim]
                r += n
                done[i] += n
            k += 1
    finally:
        lib().ingot_skv_destroy(h)
    return outs


SHAPES = {
    "plain": Shape(4, 2, 16, 16),
    "window_gate": Shape(6, 2, 44, 20, window=37, rot=24, gate="element", mix=0.3),
    "norm_gate": Shape(5, 1, 72, 40, norm="head", gate="head", mix=0.6),
    "sink": Shape(3, 3, 33, 64, norm="whole", rot=32, scaling={"factor": 3.0, "original": 40, "fast": 6.0, "slow": 1.0}, sink=True),
    "wide": Shape(8, 2, 128, 128, window=200, rot=128, sink=True, gate="element"),
    "unequal": Shape(4, 1, 192, 100, norm="whole", rot=64, gate="head"),
    "long_values": Shape(7, 1, 40, 200, window=64, sink=True, norm="head"),
    "past_the_tensor_cores": Shape(2, 1, 300, 90, rot=100, norm="head", gate="element", window=90),
    "many": Shape(40, 2, 24, 56, norm="head", rot=6, window=16, mix=1.0),
}


@pytest.mark.parametrize("name", SHAPES)
@pytest.mark.parametrize("dtype,impl", [(F32, 1), (F16, 1), (F16, 2), (F16, 3), (F16, 0)])
def test_ragged_portions(name, dtype, impl):
    s = SHAPES[name]
    if (impl == 3 and s.vdim > 128) or (impl >= 2 and s.dim > 256):
        pytest.skip("heads past the tensor-core kernels' sizes")
    rng = np.random.default_rng(3)
    w = Weights(s, 5)
    seqs = [sequence(s, n, rng) for n in (310, 47, 130, 1)]
    got = run(s, seqs, [[150, 1, 2, 77], [1, 3], [64, 66], [1]], w, dtype, impl)
    for x, y in zip(seqs, got):
        want = reference(s, x, w)
        assert np.abs(y - want).max() < (2e-5 if dtype == F32 else 6e-3) * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("dtype,impl", [(F32, 1), (F16, 2), (F16, 3)])
@pytest.mark.parametrize("window", [0, 1, 16, 17, 40, 128, 129])
def test_a_key_that_stands_out(window, dtype, impl, decoded):
    """One key has nearly all the weight wherever it is seen: just inside the window it takes over the result, just outside it is gone."""
    if decoded and impl == 3:
        pytest.skip("decoded tokens take the split-key kernel")
    s = Shape(4, 2, 32, 16, window=window, scale=1.0)
    rng = np.random.default_rng(window)
    n = 300
    x = sequence(s, n, rng)
    x[0][:] = 0.05 * x[0]
    x[1][:] = 0.05 * x[1]
    x[0][:, :, 0] = 4.0
    loud = [0, 15, 16, 127, 128, 160, 255]
    for j, at in enumerate(loud):
        x[1][at, :, 0] = 4.0 + j  # later ones are louder: each is the one that is heard while it is the latest
        x[2][at] = 10.0 * (j + 1)
    w = Weights(s)
    got = run(s, [x], [[100] + [1] * 400 if decoded else [n]], w, dtype, impl)[0]
    want = reference(s, x, w)
    assert np.abs(got - want).max() < (1e-4 if dtype == F32 else 0.06)
    if window:
        for j, at in enumerate(loud):
            others = [a for a in loud if a > at and a <= at + window]
            if at + window < n and not others:
                assert abs(got[at + window - 1].mean() - 10.0 * (j + 1)) < 1.0 and abs(got[at + window].mean() - 10.0 * (j + 1)) > 5.0


@pytest.mark.parametrize("sink", [-30.0, 0.0, 6.0, 40.0])
@pytest.mark.parametrize("dtype,impl", [(F32, 1), (F16, 2), (F16, 3)])
def test_sinks_from_nothing_to_everything(sink, dtype, impl):
    s = Shape(3, 1, 24, 24, sink=True)
    rng = np.random.default_rng(1)
    w = Weights(s)
    w.sink = np.array([sink, sink + 1, sink - 2])
    x = sequence(s, 200, rng)
    got = run(s, [x], [[130, 1, 1, 68]], w, dtype, impl)[0]
    want = reference(s, x, w)
    assert np.abs(got - want).max() < (2e-5 if dtype == F32 else 5e-3)
    assert sink < 40 or np.abs(got).max() < 1e-6


@pytest.mark.parametrize("dtype", [F32, F16])
def test_many_key_shares(dtype):
    """Thousands of keys before a few decoded tokens: the keys are split over CTAs, and one share holds the key that counts."""
    s = Shape(4, 1, 64, 32, rot=0, scale=0.6, sink=True)
    rng = np.random.default_rng(8)
    n = 5003
    x = sequence(s, n, rng)
    x[0][:, :, 1] = 3.0
    x[1][777, :, 1] = 12.0
    x[2][777] = 25.0
    w = Weights(s)
    got = run(s, [x], [[n - 3, 1, 1, 1]], w, dtype, 0)[0]
    want = reference(s, [a[:] for a in x], w)[-3:]
    assert np.abs(got[-3:] - want).max() < (1e-4 if dtype == F32 else 0.08) and np.abs(want).max() > 20


def test_rotation_far_from_the_start():
    """Scores depend on the distance only, also hundreds of thousands of positions away: one sequence, appended behind an offset."""
    import torch
    s = Shape(2, 1, 32, 16, rot=32, window=64, base=10000.0)
    rng = np.random.default_rng(0)
    x = sequence(s, 60, rng)
    outs = []
    for start in (0, 400000):
        h = C.c_void_p()
        lib(lib().ingot_skv_create_joined(C.byref(h), 1, 1, 48, F32, s.window, 8))
        turns = dev(R.frequencies(32, 10000.0)[0] / (2 * np.pi), np.float64)
        proj = dev(np.concatenate([pad(a, d) for a, (_, _, d) in zip(x, s.parts())], axis=1))
        st = Step([60], [start], [0])
        td, fd = dev([[3, 1, 0, 5]], np.int32), dev([start // 16], np.int32)
        q, out = torch.zeros(60, 2, 32, device="cuda"), torch.zeros(60, 32, device="cuda")
        o = act_out(out)
        lib(lib().ingot_gqa_append(h, 0, C.byref(st.c), proj.data_ptr(), proj.shape[1], 0, 64, 96, C.byref(s.c), None, None, EPS, turns.data_ptr(), 1.0, None, 0, 0.0, q.data_ptr(),
                                   td.data_ptr(), fd.data_ptr(), 4, None))
        # the first visible key of the first rows lies before what is held: they are left out of the comparison through the window
        s2 = CShape(2, 1, 32, 16, 32, 32, 0)
        if start == 0:
            lib(lib().ingot_gqa_attend(h, 0, C.byref(st.c), q.data_ptr(), C.byref(s2), s.scale, None, None, 0, 0, C.byref(o), td.data_ptr(), fd.data_ptr(), 4, 1, None))
        torch.cuda.synchronize()
        outs.append((q.cpu().numpy(), out.cpu().numpy()))
        lib().ingot_skv_destroy(h)
    turned = np.stack([R.rotate(x[0][t:t + 1], [400000 + t], 32, 10000.0)[0] for t in range(60)])
    assert np.abs(outs[1][0] - turned).max() < 2e-6 * np.abs(turned).max() + 2e-6
    assert np.abs(outs[0][1].reshape(60, 2, 16) - reference(s, x, Weights(s))).max() < 2e-5


def test_first_values_are_kept_for_the_later_layers():
    import torch
    s = Shape(2, 2, 16, 24, mix=0.25)
    rng = np.random.default_rng(2)
    a, b = sequence(s, 20, rng), sequence(s, 20, rng)
    h = C.c_void_p()
    lib(lib().ingot_skv_create_joined(C.byref(h), 2, 2, s.dim_p + s.vdim_p, F32, 0, 4))
    try:
        st, td, fd = Step([20], [0], [0]), dev([[2, 0]], np.int32), dev([0], np.int32)
        first = torch.full((20, 2 * s.vdim_p), float("nan"), device="cuda")
        q, out = torch.zeros(20, 2, 16, device="cuda"), torch.zeros(20, 2 * s.vdim_p, device="cuda")
        o = act_out(out)
        for layer, x in enumerate((a, b)):
            proj = dev(np.concatenate([pad(v, d) for v, (_, _, d) in zip(x, s.parts())], axis=1))
            lib(lib().ingot_gqa_append(h, layer, C.byref(st.c), proj.data_ptr(), proj.shape[1], 0, 32, 64, C.byref(s.c), None, None, EPS, None, 1.0, first.data_ptr(), int(layer == 0),
                                       0.25, q.data_ptr(), td.data_ptr(), fd.data_ptr(), 2, None))
            lib(lib().ingot_gqa_attend(h, layer, C.byref(st.c), q.data_ptr(), C.byref(s.c), s.scale, None, None, 0, 0, C.byref(o), td.data_ptr(), fd.data_ptr(), 2, 1, None))
            torch.cuda.synchronize()
            want = reference(s, x[:3] + [a[2]], Weights(s)) if layer else R.attend(x[0], x[1], x[2], s.scale)
            assert np.abs(out.cpu().numpy().reshape(20, 2, -1)[:, :, :24] - want).max() < 2e-5
    finally:
        lib().ingot_skv_destroy(h)


def test_refusals():
    h = C.c_void_p()
    lib(lib().ingot_skv_create_joined(C.byref(h), 1, 2, 48, F16, 0, 4))
    try:
        st, t = Step([3], [0], [0]), dev(np.zeros((3, 256)))
        td = dev([[0]], np.int32)
        o = act_out(t)
        good = Shape(4, 2, 32, 16)
        call = lambda c, layer=0, impl=0: lib().ingot_gqa_attend(h, layer, C.byref(st.c), t.data_ptr(), C.byref(c), 1.0, None, None, 0, 0, C.byref(o), td.data_ptr(), None, 1, impl, None)
        assert call(good.c, layer=1) == 1 and call(Shape(4, 4, 32, 16).c) == 1 and call(Shape(4, 2, 16, 16).c) == 1 and call(Shape(3, 2, 32, 16).c) == 1
        odd = CShape(4, 2, 36, 12, 36, 0, 0)
        assert call(odd, impl=2) == 3 and call(odd, impl=3) == 3
        app = lambda c: lib().ingot_gqa_append(h, 0, C.byref(st.c), t.data_ptr(), 256, 0, 128, 192, C.byref(c), None, None, EPS, None, 1.0, None, 0, 0.0, t.data_ptr(), td.data_ptr(), None, 1, None)
        assert app(Shape(4, 2, 32, 16, rot=8).c) == 1 and app(Shape(4, 2, 32, 16, norm="head").c) == 1  # no frequencies, no weights
    finally:
        lib().ingot_skv_destroy(h)
