"""Prefill and decode throughput of the sandwich-normed grouped-query attention / grouped-mixture design ("Silevik") at sizes of real
layers, beside this framework's Llama-shaped layers of equal width and heads (hybrid_bench.LlamaLayers).

Random weights. Times are device times (CUDA events around the launches of a step); the weights of a step exceed the L2.
"""
import json
import os
import statistics

import numpy as np

from . import hybrid_bench as HB
from . import models as M

SIZES = {
    # name: width, (heads, kv_heads, dim), window, dense ff, (experts, identity, top, groups, keep, ff, shared ff)
    "w2048": (2048, (16, 4, 128), 2048, 8192, (32, 8, 8, 8, 4, 1408, 1408)),
    "w4096": (4096, (32, 8, 128), 4096, 14336, (16, 4, 4, 4, 3, 3584, 3584)),
}
VOCAB = HB.VOCAB
NORMS = ("norm1", "norm1b", "norm2", "norm2b")


def config(size):
    """Windowed and full attention in turn, dense feed-forwards and mixtures in turn; one layer with scaled rotation and sinks."""
    width, (heads, kv, dim), window, ff, (experts, identity, top, groups, keep, eff, sff) = SIZES[size]
    mixer = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "v_mix": True}
    rot = {"base": 500000.0, "dims": dim}
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top, "scale": 2.0, "groups": {"count": groups, "keep": keep}},
           "expert": {"ff": eff}, "shared": {"ff": sff}}
    windowed = {"type": "attention", "mixer": dict(mixer, rot=rot, mask={"size": window}), "mlp": dense}
    full = {"type": "attention_2", "mixer": dict(mixer), "mlp": moe}
    sinks = {"type": "attention_3", "mixer": dict(mixer, rot=dict(rot, scaling={"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0})), "mlp": moe}
    return {"architecture": "Silevik", "layers": [windowed, full, windowed, sinks], "norm": {"eps": 1e-6}, "vocab": VOCAB, "width": width, "logit_scale": 0.5,
            "embedding": {"scale": float(width) ** 0.5}}


def weight_shapes(cfg):
    d = cfg["width"]
    out = {"embed": (cfg["vocab"], d), "head": (cfg["vocab"], d), "final.norm": (d,), "final.norm.b": (d,)}
    gated = lambda p, f: {p + "gate": (f, d), p + "up": (f, d), p + "down": (d, f)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, e, t = f"l{i}.", layer["mixer"], layer["mlp"], layer["type"]
        hq, hk, hv, ho = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
        for n in NORMS:
            out.update({p + n: (d,), p + n + ".b": (d,)})
        out.update({p + "mix.q": (hq, d), p + "mix.k": (hk, d), p + "mix.v": (hv, d), p + "mix.o": (d, ho), p + "mix.vmix": ()})
        if t == "attention":
            out[p + "mix.g"] = (ho, d)
        elif t == "attention_2":
            out.update({p + "mix.g": (m["heads"], d), p + "mix.q.norm": (m["dim"],), p + "mix.k.norm": (m["dim"],)})
        else:
            out.update({p + "mix.sink": (m["heads"],), p + "mix.q.norm": (hq,), p + "mix.k.norm": (hk,)})
        if e["kind"] == "dense":
            out.update(gated(p + "mlp.", e["ff"]))
        else:
            n = e["router"]["experts"] + e["router"]["identity"]
            out.update({p + "mlp.router": (n, d), p + "mlp.correction": (n,), p + "mlp.shared.sg": (1, d), **gated(p + "mlp.shared.", e["shared"]["ff"])})
            for j in range(e["router"]["experts"]):
                out.update(gated(f"{p}mlp.e{j}.", e["expert"]["ff"]))
    return out


def write_model(folder, cfg):
    import torch
    g = torch.Generator(device="cuda").manual_seed(0)
    tensors = {}
    for name, shape in weight_shapes(cfg).items():
        x = torch.randn(shape, device="cuda", generator=g)
        if "norm" in name:
            x = 0.1 * x + (0 if name.endswith(".b") else 1)
        elif name.endswith(("vmix", "correction")):
            x = 0.5 + 0.1 * x
        elif len(shape) > 1 and name != "embed":
            x = x / shape[-1] ** 0.5
        tensors[name] = ("BF16", x.bfloat16().view(torch.int16).cpu().numpy().view(np.uint16))
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    M.write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return folder


def token_params(cfg):
    """Weights a token's products read in all layers (as many experts as it can choose without an identity one), and in the output matrix."""
    d, total = cfg["width"], 0
    for layer in cfg["layers"]:
        m, e = layer["mixer"], layer["mlp"]
        hq, hk, hv, ho = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
        total += d * (hq + hk + hv + ho + {"attention": ho, "attention_2": m["heads"], "attention_3": 0}[layer["type"]])
        if e["kind"] == "dense":
            total += 3 * d * e["ff"]
        else:
            r = e["router"]
            total += d * (r["experts"] + r["identity"] + 1) + 3 * d * e["shared"]["ff"] + 3 * d * e["expert"]["ff"] * r["top"] * r["experts"] / (r["experts"] + r["identity"])
    return total, cfg["vocab"] * d


def prefill_flops(cfg, n):
    """Products of a prompt (one output row; experts at their even share), attention over what is seen."""
    layers, head = token_params(cfg)
    total = 2 * n * layers + 2 * head
    for layer in cfg["layers"]:
        m = layer["mixer"]
        seen = min(n, m["mask"]["size"]) if "mask" in m else n
        total += 2 * m["heads"] * (m["dim"] + m["vdim"]) * (seen * (seen + 1) // 2 + (n - seen) * seen)
    return total


def run_grouped(size, prefill=(512, 2048, 8192), batches=(1, 8, 32), reps=10, work="/tmp"):
    cfg = config(size)
    folder = write_model(os.path.join(work, f"ingot_grouped_{size}"), cfg)
    rng = np.random.default_rng(0)
    layers, head = token_params(cfg)
    token_bytes = 2 * (layers + head)
    out = {"layers": len(cfg["layers"]), "token_weight_gb": round(token_bytes / 1e9, 4), "prefill": {}, "decode": {}}
    with M.Model(folder, max_tokens=max(prefill) + 64, max_seqs=2, max_step_tokens=max(prefill)) as m:
        for n in prefill:
            t = rng.integers(0, VOCAB, n)
            ms = HB.step_ms(m, [(0, 0, t, [n - 1])], reps)
            out["prefill"][n] = {"ms": round(ms, 4), "tok_s": round(n / ms * 1e3), "tflops": round(prefill_flops(cfg, n) / ms / 1e9, 1)}
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
