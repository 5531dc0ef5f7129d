"""Shared-row chunked attention (csrc/attn_shared_kv.cu) through the C ABI against hybrid_reference.py: both cache types, every
kernel, head sizes that need padding, pages in random order, chunk edges with one key that stands out."""
import ctypes as C

import numpy as np
import pytest

import hybrid_reference as R
from hybrid_step import Step, act_out, dev, lib

pytestmark = pytest.mark.gpu
F32, F16 = 0, 1
EPS, OUT_SCALE = 1e-5, 0.7


def score_scale(dim):
    return 1.7 / dim ** 0.5


def reference(q, kv, wq, wk, heads, kv_heads, dim, chunk):
    n = q.shape[0]
    qn = R.rms_norm(q, wq, EPS).reshape(n, heads, dim)
    kn = R.rms_norm(kv, wk, EPS).reshape(n, kv_heads, dim)
    vis = R.chunk_visible(n, chunk) if chunk else np.tril(np.ones((n, n), bool))
    return OUT_SCALE * R.attend(qn, kn, kv.reshape(n, kv_heads, dim), score_scale(dim), vis).reshape(n, -1)


def pad_heads(a, n_heads, dim, row):
    out = np.zeros((*a.shape[:-1], n_heads, row))
    out[..., :dim] = a.reshape(*a.shape[:-1], n_heads, dim)
    return out.reshape(*a.shape[:-1], n_heads * row)


def run(seqs, cuts, heads, kv_heads, dim, chunk, dtype, wq, wk, impl, seed=0, spare=3):
    """seqs: [(q, kv)] per sequence; cuts: portion lengths per sequence. Returns the outputs per sequence."""
    import torch
    rng = np.random.default_rng(seed)
    row = (dim + 7) // 8 * 8 if dtype == F32 else lib().ingot_skv_row_length(dim)
    pages = [lib().ingot_skv_pages(chunk, q.shape[0]) for q, _ in seqs]
    order = rng.permutation(sum(pages) + spare).astype(np.int32)
    tables, at = [], 0
    for p in pages:
        tables.append(order[at:at + p])
        at += p
    h = C.c_void_p()
    lib(lib().ingot_skv_create(C.byref(h), 2, kv_heads, row, dtype, chunk, len(order)))
    wqd, wkd = dev(pad_heads(wq, heads, dim, row)), dev(pad_heads(wk, kv_heads, dim, row))
    outs = [np.zeros((q.shape[0], heads * dim)) for q, _ in seqs]
    done = [0] * len(seqs)
    k = 0
    try:
        while any(d < q.shape[0] for d, (q, _) in zip(done, seqs)):
            live = [i for i, (q, _) in enumerate(seqs) if done[i] < q.shape[0]]
            part = [min(cuts[i][k % len(cuts[i])], seqs[i][0].shape[0] - done[i]) for i in live]
            st = Step(part, [done[i] for i in live], [0] * len(live))
            proj = np.concatenate([np.concatenate([pad_heads(seqs[i][0][done[i]:done[i] + n], heads, dim, row),
                                                   pad_heads(seqs[i][1][done[i]:done[i] + n], kv_heads, dim, row)], axis=1)
                                   for i, n in zip(live, part)])
            pd = dev(proj)
            # tables hold only the pages from the first visible one on
            first = [lib().ingot_skv_pages(chunk, (done[i] // chunk * chunk if chunk else 0) + 1) - 1 for i in live]
            width = max(len(tables[i]) - f for i, f in zip(live, first))
            tab = np.full((len(live), width), -1, np.int32)
            for r, (i, f) in enumerate(zip(live, first)):
                tab[r, :len(tables[i]) - f] = tables[i][f:]
            td, fd = dev(tab, np.int32), dev(first, np.int32)
            q_out = torch.zeros(st.n_tok, heads, row, device="cuda", dtype=torch.float32 if dtype == F32 else torch.float16)
            out = torch.zeros(st.n_tok, heads * dim, device="cuda")
            o = act_out(out)
            for layer in (0, 1):  # layer 1 holds the same rows and must not disturb layer 0
                lib(lib().ingot_skv_append(h, layer, C.byref(st.c), pd.data_ptr(), proj.shape[1], 0, heads * row, heads, dim, wqd.data_ptr(),
                                           wkd.data_ptr(), EPS, q_out.data_ptr(), td.data_ptr(), fd.data_ptr(), width, None))
            lib(lib().ingot_skv_attend(h, 0, C.byref(st.c), q_out.data_ptr(), heads, dim, score_scale(dim), OUT_SCALE, C.byref(o), td.data_ptr(),
                                       fd.data_ptr(), width, impl, None))
            torch.cuda.synchronize()
            status = C.c_int(-1)
            lib(lib().ingot_skv_status(h, None, C.byref(status)))
            assert status.value == 0
            r = 0
            for i, n in zip(live, part):
                outs[i][done[i]:done[i] + n] = out[r:r + n].cpu().numpy()
                r += n
                done[i] += n
            k += 1
    finally:
        lib().ingot_skv_destroy(h)
    return outs


CUTS = {"whole": [[10 ** 9]] * 3, "portions": [[70, 2, 33, 16], [5, 64], [2]], "single": [[1]] * 3}
SHAPES = [(10, 2, 64, 48), (4, 4, 24, 40), (8, 2, 128, 0), (12, 3, 20, 33), (16, 2, 80, 100), (2, 1, 256, 64), (20, 1, 16, 16), (5, 5, 96, 7)]


@pytest.mark.parametrize("cut", CUTS)
@pytest.mark.parametrize("heads,kv_heads,dim,chunk", SHAPES)
@pytest.mark.parametrize("dtype,impl", [(F32, 0), (F16, 1), (F16, 2), (F16, 0)])
def test_against_plain_attention(heads, kv_heads, dim, chunk, cut, dtype, impl):
    rng = np.random.default_rng(heads * dim)
    wq, wk = 1 + 0.3 * rng.standard_normal(heads * dim), 1 + 0.3 * rng.standard_normal(kv_heads * dim)
    seqs = [(rng.standard_normal((n, heads * dim)), 2 * rng.standard_normal((n, kv_heads * dim))) for n in (137, 67, 3)]
    got = run(seqs, CUTS[cut], heads, kv_heads, dim, chunk, dtype, wq, wk, impl)
    for (q, kv), g in zip(seqs, got):
        want = reference(q, kv, wq, wk, heads, kv_heads, dim, chunk)
        assert np.abs(g - want).max() < (2e-5 if dtype == F32 else 8e-3), np.abs(g - want).max()


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("dtype,impl", [(F32, 0), (F16, 1), (F16, 2), (F16, 0)])
def test_a_key_that_stands_out_is_seen_up_to_the_chunks_edge_and_not_beyond(dtype, impl, decoded):
    """One query matches one key so strongly that it takes all the weight if it is visible; the key sits at the first and at the
    last place of a chunk, at page borders, and the query just inside and just outside."""
    heads, kv_heads, dim, chunk, n = 4, 1, 32, 40, 130
    rng = np.random.default_rng(5)
    ones_q, ones_k = np.ones(heads * dim), np.ones(kv_heads * dim)
    for key, query in [(0, 39), (0, 40), (39, 39), (39, 40), (40, 79), (40, 80), (55, 56), (56, 72), (79, 80), (80, 119), (15, 39), (16, 40), (80, 120)]:
        q = 0.05 * rng.standard_normal((n, heads * dim))
        kv = 0.05 * rng.standard_normal((n, dim)) + np.eye(dim)[rng.integers(1, dim, n)]
        kv[key] = 6 * np.eye(dim)[0]
        q[query] = np.tile(9 * np.eye(dim)[0], heads)
        want = reference(q, kv, ones_q, ones_k, heads, kv_heads, dim, chunk)
        cuts = [[query, 1, 10 ** 9]] if decoded else [[10 ** 9]]
        got = run([(q, kv)], cuts, heads, kv_heads, dim, chunk, dtype, ones_q, ones_k, impl)[0]
        seen = key // chunk == query // chunk
        assert (got[query, 0] > 0.9 * OUT_SCALE * 6) == seen, (key, query)
        assert np.abs(got - want).max() < (2e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("heads,kv_heads,dim,chunk", [(8, 2, 128, 0), (4, 4, 112, 96), (6, 1, 128, 200), (16, 2, 100, 33), (3, 1, 126, 1000)])
def test_tcgen05_kernel(heads, kv_heads, dim, chunk):
    """Rows of 128 values on the tcgen05 kernel: several row tiles, unequal sequences, portions that start inside chunks and
    pages, single tokens beside long portions."""
    rng = np.random.default_rng(heads + dim)
    wq, wk = 1 + 0.3 * rng.standard_normal(heads * dim), 1 + 0.3 * rng.standard_normal(kv_heads * dim)
    seqs = [(rng.standard_normal((n, heads * dim)), 2 * rng.standard_normal((n, kv_heads * dim))) for n in (700, 300, 5)]
    for cuts in ([[10 ** 9]] * 3, [[133, 1, 300], [7, 90, 1], [1]]):
        got = run(seqs, cuts, heads, kv_heads, dim, chunk, F16, wq, wk, 3)
        for (q, kv), g in zip(seqs, got):
            want = reference(q, kv, wq, wk, heads, kv_heads, dim, chunk)
            assert np.abs(g - want).max() < 8e-3, np.abs(g - want).max()


@pytest.mark.parametrize("heads,kv_heads,dim,chunk,n", [(8, 2, 128, 0, 1500), (7, 1, 64, 900, 2000), (32, 1, 32, 0, 700), (4, 2, 200, 0, 600)])
def test_decoding_over_many_keys(heads, kv_heads, dim, chunk, n):
    """Single tokens after long prompts: keys split over several thread blocks, unequal sequences in the batch, more heads than
    one row tile."""
    rng = np.random.default_rng(n)
    wq, wk = 1 + 0.3 * rng.standard_normal(heads * dim), 1 + 0.3 * rng.standard_normal(kv_heads * dim)
    seqs = [(rng.standard_normal((m, heads * dim)), 2 * rng.standard_normal((m, kv_heads * dim))) for m in (n, n // 3, 9)]
    cuts = [[n - 3, 1, 1, 1], [n // 3 - 3, 1, 1, 1], [6, 1, 1, 1]]
    got = run(seqs, cuts, heads, kv_heads, dim, chunk, F16, wq, wk, 0)
    for (q, kv), g in zip(seqs, got):
        want = reference(q[:], kv, wq, wk, heads, kv_heads, dim, chunk)
        assert np.abs(g[-3:] - want[-3:]).max() < 8e-3, np.abs(g - want).max()


def test_a_table_entry_outside_the_pool_is_reported():
    import torch
    h = C.c_void_p()
    lib(lib().ingot_skv_create(C.byref(h), 1, 1, 16, F32, 32, 4))
    st = Step([3], [0], [0])
    proj, w, tab = dev(np.ones((3, 32))), dev(np.ones(16)), dev([[7, 1]], np.int32)  # block 7 of a pool of 4
    q_out, out = torch.zeros(3, 16, device="cuda"), torch.zeros(3, 16, device="cuda")
    lib(lib().ingot_skv_append(h, 0, C.byref(st.c), proj.data_ptr(), 32, 0, 16, 1, 16, w.data_ptr(), w.data_ptr(), EPS, q_out.data_ptr(),
                               tab.data_ptr(), None, 2, None))
    status = C.c_int(0)
    lib(lib().ingot_skv_status(h, None, C.byref(status)))
    assert status.value == 2
    lib(lib().ingot_skv_status(h, None, C.byref(status)))
    assert status.value == 0
    lib().ingot_skv_destroy(h)
