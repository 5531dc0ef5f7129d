"""Prefill and decode throughput of the latent-attention / mixture-of-experts design ("Banevik") at sizes of real layers, beside this
framework's Llama-shaped layers of equal width and heads (hybrid_bench.LlamaLayers).

Random weights. Times are device times (CUDA events around the launches of a step); the weights of a step exceed the L2.
"""
import json
import os
import statistics

import numpy as np

from . import hybrid_bench as HB
from . import models as M

SIZES = {
    # name: width, heads, (dim, rot_dim, vdim, kv_rank), window, (experts, top, ff)
    "w2048": (2048, 16, (128, 64, 128, 512), 2048, (32, 8, 1408)),
    "w4096": (4096, 32, (128, 64, 128, 512), 4096, (16, 4, 3584)),
}
VOCAB = HB.VOCAB
RUNS = 4  # three layers, the middle one twice


def config(size):
    width, heads, (dim, rot, vdim, rank), window, (experts, top, ff) = SIZES[size]
    layer = {"type": "latent_attention", "mlp": {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}},
             "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": (dim + rot) ** -0.5, "rot": {"base": 500000.0, "dims": rot},
                       "mask": {"size": window}}}
    return {"architecture": "Banevik", "layers": [layer] * 3, "loop": {"start": 1, "stop": 2, "times": 2}, "norm": {"eps": 1e-6}, "vocab": VOCAB, "width": width,
            "logit_softcap": 30.0, "embedding": {"bigram": {"buckets": 65521, "mul_prev": 1009, "mul_cur": 8191}}}


def weight_shapes(cfg):
    d = cfg["width"]
    out = {"embed": (cfg["vocab"], d), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, d), "loop.in": (d, 2 * d), "final.norm": (d,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, e = f"l{i}.", layer["mixer"], layer["mlp"]
        H, k, r, v, c, f = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], e["expert"]["ff"]
        out.update({p + "norm1": (d,), p + "norm2": (d,), p + "mix.q": (H * (k + r), d), p + "mix.dkv": (c + r, d), p + "mix.dkv.norm": (c,), p + "mix.uk": (H * k, c),
                    p + "mix.uv": (H * v, c), p + "mix.sink": (H,), p + "mix.o": (d, H * v), p + "mlp.router": (e["router"]["experts"], d)})
        for j in range(e["router"]["experts"]):
            out.update({f"{p}mlp.e{j}.up": (f, d), f"{p}mlp.e{j}.down": (d, f)})
    return out


def write_model(folder, cfg):
    import torch
    g = torch.Generator(device="cuda").manual_seed(0)
    tensors = {}
    for name, shape in weight_shapes(cfg).items():
        x = torch.randn(shape, device="cuda", generator=g)
        if "norm" in name:
            x = 0.1 * x + (1 if name.endswith("dkv.norm") else 0)
        elif len(shape) > 1 and name not in ("embed", "bigram"):
            x = x / shape[-1] ** 0.5
        tensors[name] = ("BF16", x.bfloat16().view(torch.int16).cpu().numpy().view(np.uint16))
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    M.write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return folder


def token_params(size):
    """Weights a token's products read in one layer run, in the loop's input product, and in the output matrix."""
    d, H, (k, r, v, c), _, (experts, top, f) = SIZES[size]
    return d * (H * (k + r) + c + r) + H * (k + v) * c + H * v * d + d * experts + 2 * top * d * f, 2 * d * d, VOCAB * d


def prefill_flops(size, n):
    """Products of a prompt (one output row), attention with keys of their own inside the window."""
    _, H, (k, r, v, _), window, _ = SIZES[size]
    layer, loop, head = token_params(size)
    full = min(n, window)
    pairs = full * (full + 1) // 2 + (n - full) * window
    return RUNS * (2 * n * layer + 2 * H * (k + r + v) * pairs) + 2 * (2 * n * loop) + 2 * head


def run_latent(size, prefill=(512, 2048, 8192), batches=(1, 8, 32), reps=10, work="/tmp"):
    cfg = config(size)
    folder = write_model(os.path.join(work, f"ingot_latent_{size}"), cfg)
    rng = np.random.default_rng(0)
    layer, loop, head = token_params(size)
    token_bytes = 2 * (RUNS * layer + 2 * loop + head)
    out = {"layer_runs": RUNS, "token_weight_gb": round(token_bytes / 1e9, 4), "prefill": {}, "decode": {}}
    with M.Model(folder, max_tokens=max(prefill) + 64, max_seqs=2, max_step_tokens=max(prefill)) as m:
        for n in prefill:
            t = rng.integers(0, VOCAB, n)
            ms = HB.step_ms(m, [(0, 0, t, [n - 1])], reps)
            out["prefill"][n] = {"ms": round(ms, 4), "tok_s": round(n / ms * 1e3), "tflops": round(prefill_flops(size, n) / ms / 1e9, 1)}
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
            out["decode"][b] = {"ms": round(ms, 4), "tok_s": round(b / ms * 1e3, 1)}
            if b == 1:
                out["decode"][b]["weight_gb_s"] = round(token_bytes / ms / 1e6, 1)
    return out
