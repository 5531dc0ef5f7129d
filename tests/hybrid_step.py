"""Device-side step descriptions for the kernel tests: the structs of include/ingot_cuda.h filled from Python lists."""
import ctypes as C

import numpy as np

import ingot_b200 as ib


class CStep(C.Structure):
    _fields_ = [("n_tok", C.c_int), ("n_seq", C.c_int), ("max_len", C.c_int), ("row_seq", C.c_void_p), ("row_start", C.c_void_p),
                ("len", C.c_void_p), ("pos0", C.c_void_p), ("slot", C.c_void_p)]


class CPlan(C.Structure):
    _fields_ = [("n_chunks", C.c_int), ("max_chunks", C.c_int), ("chunk_seq", C.c_void_p), ("chunk_t0", C.c_void_p), ("chunk_len", C.c_void_p),
                ("seq_chunk0", C.c_void_p), ("scratch_dev", C.c_void_p), ("scratch_floats", C.c_size_t)]


class CActOut(C.Structure):
    _fields_ = [("f32", C.c_void_p), ("hi", C.c_void_p), ("lo", C.c_void_p), ("ld", C.c_int)]


def dev(x, dtype=np.float32):
    """A numpy array as a (canary-guarded) device tensor."""
    import torch
    src = torch.from_numpy(np.ascontiguousarray(x, dtype=dtype))
    t = ib.guarded_empty(src.shape, src.dtype)
    t.copy_(src)
    return t


def lib(rc=None):
    """lib() is the library; lib(rc) checks a status."""
    if rc is None:
        return ib.lib()
    ib._check(rc)


class Step:
    def __init__(self, lens, pos0, slots):
        self.n_tok = int(sum(lens))
        start = np.concatenate([[0], np.cumsum(lens)[:-1]])
        self.keep = [dev(a, np.int32) for a in (np.repeat(np.arange(len(lens)), lens), start, lens, pos0, slots)]
        self.c = CStep(self.n_tok, len(lens), int(max(lens)), *[t.data_ptr() for t in self.keep])


class plan:
    def __init__(self, lens, run, scratch_per_chunk):
        import torch
        seq, t0, ln, first, most = [], [], [], [], 1
        for i, n in enumerate(lens):
            first.append(len(seq))
            for t in range(0, n, run):
                seq.append(i)
                t0.append(t)
                ln.append(min(run, n - t))
            most = max(most, len(seq) - first[-1])
        first.append(len(seq))
        self.keep = [dev(a, np.int32) for a in (seq, t0, ln, first)]
        self.scratch = ib.guarded_empty((len(seq) * scratch_per_chunk,), torch.float32)
        self.c = CPlan(len(seq), most, *[t.data_ptr() for t in self.keep], self.scratch.data_ptr(), self.scratch.numel())


def act_out(f32=None, hi=None, lo=None):
    some = f32 if f32 is not None else hi
    ptr = lambda t: None if t is None else t.data_ptr()
    return CActOut(ptr(f32), ptr(hi), ptr(lo), some.shape[-1])
