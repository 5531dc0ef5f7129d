"""Small random models of the looped latent-attention / mixture-of-experts design for the tests: configurations, weights, and
the plain implementation's logits (folders are written by hybrid_models.write)."""
import numpy as np

import latent_moe_reference as R
from ingot_b200 import models as M


def layer(heads, dim, rot_dim, vdim, kv_rank, window, scale=0.2, base=10000.0, experts=None, top=1, ff=24, rot_dims=None):
    mlp = None if experts is None else {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim if rot_dims is None else rot_dims}, "mask": {"size": window}}}


def config(layers, vocab=96, width=48, eps=1e-5, loop=None, bigram=None, softcap=9.0):
    cfg = {"architecture": "Banevik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_softcap": softcap,
           "embedding": {"bigram": None if bigram is None else dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))},
           "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))}
    return cfg


def shapes(cfg):
    d = cfg["width"]
    out = {"embed": (cfg["vocab"], d), "final.norm": (d,)}
    if cfg["embedding"]["bigram"]:
        out["bigram"] = (cfg["embedding"]["bigram"]["buckets"] + 1, d)
    if cfg["loop"]:
        out["loop.in"] = (d, 2 * d)
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}."
        H, k, r, v, c = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        out.update({p + "norm1": (d,), p + "mix.q": (H * (k + r), d), p + "mix.dkv": (c + r, d), p + "mix.dkv.norm": (c,), p + "mix.uk": (H * k, c),
                    p + "mix.uv": (H * v, c), p + "mix.sink": (H,), p + "mix.o": (d, H * v)})
        if spec["mlp"]:
            f = spec["mlp"]["expert"]["ff"]
            out.update({p + "norm2": (d,), p + "mlp.router": (spec["mlp"]["router"]["experts"], d)})
            for e in range(spec["mlp"]["router"]["experts"]):
                out.update({f"{p}mlp.e{e}.up": (f, d), f"{p}mlp.e{e}.down": (d, f)})
    return out


def random_weights(cfg, seed=0):
    """bf16-representable float32 weights. Scores are sharp and sinks matter, so that a key on the wrong side of a window's edge, a
    sink left out or a wrong expert moves the logits."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in shapes(cfg).items():
        x = rng.standard_normal(shape)
        if name.endswith(("norm", "norm1", "norm2")):
            x = 0.25 * x + (1.0 if name.endswith("dkv.norm") else 0.0)
        elif name.endswith("sink"):
            x = x + 2.0
        elif name == "embed":
            x = x * 0.5
        elif name != "bigram":
            x = x / np.sqrt(shape[-1])
            if name.endswith(("mix.q", "mix.dkv")):
                x = x * 2.0
            elif name.endswith("router"):
                x = x * 3.0
            elif name.endswith(".down"):
                x = x * 0.7
        w[name] = M.from_bf16(M.to_bf16(x))
    return w


def reference_logits(cfg, weights, tokens, residuals=None):
    return R.forward(tokens, {k: v.astype(np.float64) for k, v in weights.items()}, cfg, residuals)


def clear_choices(cfg, weights, tokens, gap=0.2):
    """[n] bool: positions at which every router's choice is clear (the best expert left out is `gap` behind, in logits)."""
    W = {k: v.astype(np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    clear = np.ones(len(tokens), bool)
    x0 = x = R.embed(tokens, W, cfg)
    for i, entry in R.layer_runs(cfg):
        p, mlp = f"l{i}.", cfg["layers"][i]["mlp"]
        if entry:
            x = np.concatenate([x, x0], axis=1) @ W["loop.in"].T
        if mlp and mlp["router"]["top"] < mlp["router"]["experts"]:
            z = np.sort(R.offset_norm(x, W[p + "norm2"], eps) @ W[p + "mlp.router"].T, axis=1)[:, ::-1]
            clear &= z[:, mlp["router"]["top"] - 1] - z[:, mlp["router"]["top"]] > gap
        x = R.layer(x, W, p, cfg, i, eps)
    return clear
