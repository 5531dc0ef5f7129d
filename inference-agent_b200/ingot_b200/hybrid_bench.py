"""Prefill and decode throughput of the hybrid design ("Besudra") at sizes of real layers, beside this framework's Llama-shaped
layers of equal width driven through the same library entry points CudaBackend makes (backend/cuda_backend.cpp: encode_layers).

Random weights. Times are device times (CUDA events around the launches of a step); the weights of a step exceed the L2.
"""
import ctypes as C
import json
import os
import statistics

import numpy as np

from . import models as M

SIZES = {
    # name: width, (inner, state, dt_rank), (heads, kv_heads, dim, chunk), (rec width, blocks), ff
    "w2048": (2048, (4096, 16, 128), (16, 4, 128, 2048), (2048, 8), 8192),
    "w4096": (4096, (8192, 16, 256), (32, 8, 128, 4096), (4096, 16), 14336),
}
VOCAB, PERIOD = 32768, 4  # three selective-scan layers, then a parallel layer with a feed-forward


def config(size, n_layer=PERIOD):
    width, (inner, state, rank), (heads, kv, dim, chunk), (rec, blocks), ff = SIZES[size]
    mamba = {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": rank, "conv": 4}, "mlp": None}
    par = {"type": "parallel",
           "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": chunk}},
                     "right": {"width": rec, "blocks": blocks, "conv": 4}, "left_scale": 0.5, "right_scale": 0.5},
           "mlp": {"kind": "dense", "ff": ff}}
    return {"architecture": "Besudra", "layers": [par if i % PERIOD == PERIOD - 1 else mamba for i in range(n_layer)], "norm": {"eps": 1e-6},
            "vocab": VOCAB, "width": width}


def weight_shapes(cfg):
    d = cfg["width"]
    out = {"embed": (cfg["vocab"], d), "head": (cfg["vocab"], d), "final.norm": (d,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        out[p + "norm1"] = (d,)
        if layer["type"] == "mamba1":
            n, s, r = m["inner"], m["state"], m["dt_rank"]
            out.update({p + "mix.in": (2 * n, d), p + "mix.conv": (n, m["conv"]), p + "mix.conv.b": (n,), p + "mix.x": (r + 2 * s, n),
                        p + "mix.dt": (n, r), p + "mix.dt.b": (n,), p + "mix.A_log": (n, s), p + "mix.D": (n,), p + "mix.o": (d, n)})
        else:
            a, b, q = m["left"], m["right"], p + "mix."
            hq, hk, w = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], b["width"]
            k = w // b["blocks"]
            out.update({q + "left.q": (hq, d), q + "left.k": (hk, d), q + "left.q.norm": (hq,), q + "left.k.norm": (hk,), q + "left.o": (d, hq),
                        q + "right.y": (w, d), q + "right.y.b": (w,), q + "right.x": (w, d), q + "right.x.b": (w,),
                        q + "right.conv": (w, b["conv"]), q + "right.conv.b": (w,), q + "right.ra": (b["blocks"], k, k),
                        q + "right.ra.b": (b["blocks"], k), q + "right.ri": (b["blocks"], k, k), q + "right.ri.b": (b["blocks"], k),
                        q + "right.lam": (w,), q + "right.o": (d, w)})
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            out.update({p + "norm2": (d,), p + "mlp.gate": (f, d), p + "mlp.up": (f, d), p + "mlp.down": (d, f)})
    return out


def write_model(folder, cfg):
    import torch
    g = torch.Generator(device="cuda").manual_seed(0)
    tensors = {}
    for name, shape in weight_shapes(cfg).items():
        x = torch.randn(shape, device="cuda", generator=g)
        if "norm" in name:
            x = 1 + 0.1 * x
        elif name.endswith("dt.b"):
            x = x - 3
        elif len(shape) > 1 and not name.endswith(("conv", "A_log")) and name != "embed":
            x = x / shape[-1] ** 0.5
        tensors[name] = ("BF16", x.bfloat16().view(torch.int16).cpu().numpy().view(np.uint16))
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    M.write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return folder


def prefill_flops(cfg, n):
    """Products, attention inside chunks (both products, causal half), scan and gates left out."""
    d, total = cfg["width"], 0
    for layer in cfg["layers"]:
        m = layer["mixer"]
        if layer["type"] == "mamba1":
            total += 2 * n * (3 * m["inner"] * d + m["inner"] * (2 * m["dt_rank"] + 2 * m["state"]))
        else:
            a, b = m["left"], m["right"]
            hq, hk, w = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], b["width"]
            total += 2 * n * (d * (2 * hq + hk + 3 * w) + 2 * w * w // b["blocks"])
            full, rest = divmod(n, a["mask"]["size"])
            total += 2 * hq * (full * a["mask"]["size"] ** 2 + rest ** 2)
        if layer["mlp"]:
            total += 2 * n * 3 * d * layer["mlp"]["ff"]
    return total


def step_ms(model, portions, reps, warmup=3):
    times = []
    for i in range(warmup + reps):
        model.step(portions)
        if i >= warmup:
            times.append(model.last_step_ms)
    return statistics.median(times)


def run_hybrid(size, prefill=(512, 2048, 8192), batches=(1, 8, 32), reps=10, work="/tmp"):
    cfg = config(size)
    folder = write_model(os.path.join(work, f"ingot_hybrid_{size}"), cfg)
    rng = np.random.default_rng(0)
    out = {"layers": len(cfg["layers"]), "prefill": {}, "decode": {}}
    with M.Model(folder, max_tokens=max(prefill) + 64, max_seqs=2, max_step_tokens=max(prefill)) as m:
        for n in prefill:
            t = rng.integers(0, VOCAB, n)
            ms = step_ms(m, [(0, 0, t, [n - 1])], reps)
            out["prefill"][n] = {"ms": round(ms, 4), "tok_s": round(n / ms * 1e3), "tflops": round(prefill_flops(cfg, n) / ms / 1e9, 1)}
        m.release(0)
        out["weight_gb"] = round(m.weight_bytes / 1e9, 4)
    ctx = 1024
    with M.Model(folder, max_tokens=(ctx + 64) * max(batches), max_seqs=max(batches), max_step_tokens=2048) as m:
        for s in range(max(batches)):
            m.step([(s, 0, rng.integers(0, VOCAB, ctx), [])])
        pos = {s: ctx for s in range(max(batches))}
        for b in batches:
            times = []
            for i in range(4 + reps):
                m.step([(s, pos[s], [int(rng.integers(0, VOCAB))], [0]) for s in range(b)])
                for s in range(b):
                    pos[s] += 1
                if i >= 4:
                    times.append(m.last_step_ms)
            ms = statistics.median(times)
            out["decode"][b] = {"ms": round(ms, 4), "tok_s": round(b / ms * 1e3, 1), "weight_gb_s": round(m.weight_bytes / ms / 1e6, 1)}
    return out


class LlamaLayers:
    """Llama-shaped layers (f16 weights, RoPE, causal GQA, SwiGLU) as CudaBackend runs them, with the same output matrix."""

    def __init__(self, size, n_layer=PERIOD, max_tok=8192, max_seqs=1):
        import torch
        import ingot_b200 as ib
        self.ib, self.torch = ib, torch
        self.width, _, (self.h, self.hkv, self.d, _), _, self.ff = SIZES[size]
        self.L = M.lib()
        P, I = C.c_void_p, C.c_int
        L = self.L
        L.ingot_linear_ws_create.argtypes = [C.POINTER(P), I, I]
        L.ingot_linear_ws_destroy.argtypes = [P]
        L.ingot_linear_tc_prepare.argtypes = [P, P, I, I, P]
        L.ingot_linear_tc_prepare_norm.argtypes = [P, P, P, C.c_float, I, I, P]
        L.ingot_linear_tc_run_partial_group.argtypes = [P, C.POINTER(P), I, C.POINTER(I), I, I, I, P]
        L.ingot_linear_tc_finish_group.argtypes = [P, C.POINTER(P), I, P]
        L.ingot_linear_tc_finish_residual_norm.argtypes = [P, P, P, C.c_float, I, P]
        L.ingot_linear_tc_finish_swiglu.argtypes = [P, I, I, P]
        L.ingot_support_linear.argtypes = [P, P, I, P, I, I, I, I, P]
        L.ingot_support_gemv_group.argtypes = [C.POINTER(P), C.POINTER(P), C.POINTER(P), I, C.POINTER(I), I, I, P, P, C.c_float, I, I, P]
        g = torch.Generator(device="cuda").manual_seed(1)
        mat = lambda n_out, n_in: (torch.randn(n_out, n_in, device="cuda", generator=g) / n_in ** 0.5).half()
        q, kv, w, ff = self.h * self.d, self.hkv * self.d, self.width, self.ff
        self.layers = [dict(q=mat(q, w), k=mat(kv, w), v=mat(kv, w), o=mat(w, q), gate=mat(ff, w), up=mat(ff, w), down=mat(w, ff)) for _ in range(n_layer)]
        self.head = mat(VOCAB, w)
        self.norm = torch.ones(w, device="cuda")
        f = lambda n: torch.zeros(max_tok, n, device="cuda")
        self.x, self.qb, self.kb, self.vb, self.ab, self.gb = f(w), f(q), f(kv), f(kv), f(q), f(ff)
        self.qr = torch.zeros(max_tok, q, device="cuda", dtype=torch.float16)
        self.logits = torch.zeros(VOCAB, device="cuda")
        self.inv = 1.0 / (500000.0 ** (torch.arange(0, self.d, 2, device="cuda") / self.d))
        self.kv = ib.KVCache(ib.KV_CONTIGUOUS, n_layer, self.hkv, max_tok)
        self.ws = C.c_void_p()
        if L.ingot_linear_ws_create(C.byref(self.ws), max_tok, max(w, ff, q)) != 0:
            raise RuntimeError("linear workspace")
        self.weight_bytes = 2 * (self.head.numel() + sum(t.numel() for l in self.layers for t in l.values()))

    def close(self):
        self.L.ingot_linear_ws_destroy(self.ws)
        self.kv.close()

    def flops(self, n):
        q, kv, w, ff = self.h * self.d, self.hkv * self.d, self.width, self.ff
        return len(self.layers) * (2 * n * (w * (2 * q + 2 * kv) + 3 * w * ff) + 2 * q * n * n)

    def encode(self, n, pos):
        L, ib = self.L, self.ib
        s = C.c_void_p(self.torch.cuda.current_stream().cuda_stream)
        p = lambda t: t.data_ptr()
        ptrs = lambda ts: (C.c_void_p * len(ts))(*[t.data_ptr() for t in ts])
        ints = lambda v: (C.c_int * len(v))(*v)
        abi = ib.lib()
        w, q, kv, ff, eps = self.width, self.h * self.d, self.hkv * self.d, self.ff, 1e-5
        ok = lambda rc: rc == 0 or (_ for _ in ()).throw(RuntimeError(f"llama layer launch failed: {rc}"))
        gemv = lambda outs, ws, rows, swiglu, x, norm, n_in, acc: ok(L.ingot_support_gemv_group(
            ptrs(outs), ptrs(ws), None, 0, ints(rows), len(ws), swiglu, p(x), p(norm) if norm is not None else None, eps, n_in, acc, s))
        for i, l in enumerate(self.layers):
            if n == 1:
                gemv([self.qb, self.kb, self.vb], [l["q"], l["k"], l["v"]], [q, kv, kv], 0, self.x, self.norm, w, 0)
            else:
                if i == 0:
                    ok(L.ingot_linear_tc_prepare_norm(self.ws, p(self.x), p(self.norm), eps, w, n, s))
                ok(L.ingot_linear_tc_run_partial_group(self.ws, ptrs([l["q"], l["k"], l["v"]]), w, ints([q, kv, kv]), 3, 0, 0, s))
                ok(L.ingot_linear_tc_finish_group(self.ws, ptrs([self.qb, self.kb, self.vb]), 3, s))
            ok(abi.ingot_rope_kv_append(self.kv.handle, i, p(self.qb), p(self.qr), p(self.kb), p(self.vb), p(self.inv), self.h, pos, n, None, None, None, 0, s))
            if n == 1:
                ok(abi.ingot_attn_decode(self.kv.handle, i, p(self.qr), ib.F16, p(self.ab), ib.F32, self.h, 1, None, pos + 1, None, 0, 0, s))
                gemv([self.x], [l["o"]], [w], 0, self.ab, None, q, 1)
                gemv([self.gb, self.gb], [l["gate"], l["up"]], [ff, ff], 1, self.x, self.norm, w, 0)
                # the streaming kernel stages rows of up to 12032 values; longer ones take the plain one, as in CudaBackend
                if ff <= 12032:
                    gemv([self.x], [l["down"]], [w], 0, self.gb, None, ff, 1)
                else:
                    ok(L.ingot_support_linear(p(self.x), p(l["down"]), 1, p(self.gb), ff, w, 1, 1, s))
            else:
                ok(abi.ingot_attn_prefill(self.kv.handle, i, p(self.qr), ib.F16, p(self.ab), ib.F32, self.h, pos, n, None, 0, s))
                ok(L.ingot_linear_tc_prepare(self.ws, p(self.ab), q, n, s))
                ok(L.ingot_linear_tc_run_partial_group(self.ws, ptrs([l["o"]]), q, ints([w]), 1, 0, 0, s))
                ok(L.ingot_linear_tc_finish_residual_norm(self.ws, p(self.x), p(self.norm), eps, 0, s))
                ok(L.ingot_linear_tc_run_partial_group(self.ws, ptrs([l["gate"], l["up"]]), w, ints([ff, ff]), 2, 0, 0, s))
                ok(L.ingot_linear_tc_finish_swiglu(self.ws, 0, 1, s))
                ok(L.ingot_linear_tc_run_partial_group(self.ws, ptrs([l["down"]]), ff, ints([w]), 1, 0, 0, s))
                last = i + 1 == len(self.layers)
                ok(L.ingot_linear_tc_finish_residual_norm(self.ws, p(self.x), None if last else p(self.norm), eps, 0, s))
        ok(L.ingot_support_gemv_group(ptrs([self.logits]), ptrs([self.head]), None, 0, ints([VOCAB]), 1, 0, p(self.x) + (n - 1) * w * 4, p(self.norm), eps, w, 0, s))

    def time(self, n, pos, reps):
        """Median device ms of one step, replayed as a CUDA graph (as CudaBackend replays its single-token step)."""
        torch = self.torch
        self.x.normal_()
        stream = torch.cuda.Stream()
        with torch.cuda.stream(stream):
            self.encode(n, pos)
            stream.synchronize()
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph, stream=stream):
                self.encode(n, pos)
            times = []
            for i in range(3 + reps):
                a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                a.record(stream)
                graph.replay()
                b.record(stream)
                stream.synchronize()
                self.x.normal_()
                if i >= 3:
                    times.append(a.elapsed_time(b))
        assert self.kv.status() == 0
        return statistics.median(times)


def run_llama(size, prefill=(512, 2048, 8192), reps=10):
    m = LlamaLayers(size, max_tok=max(prefill))
    out = {"layers": len(m.layers), "weight_gb": round(m.weight_bytes / 1e9, 4), "prefill": {}, "decode": {}}
    for n in prefill:
        ms = m.time(n, 0, reps)
        out["prefill"][n] = {"ms": round(ms, 4), "tok_s": round(n / ms * 1e3), "tflops": round(m.flops(n) / ms / 1e9, 1)}
    ms = m.time(1, 1024, reps)
    out["decode"][1] = {"ms": round(ms, 4), "tok_s": round(1e3 / ms, 1), "weight_gb_s": round(m.weight_bytes / ms / 1e6, 1)}
    m.close()
    return out
