"""Small random models of the sandwich-normed attention / grouped-mixture design for the tests: configurations, weights, and the plain
implementation's logits (folders are written by hybrid_models.write)."""
import numpy as np

import silevik_reference as R
from ingot_b200 import models as M


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, groups, ff, shared, scale=1.5):
    """groups: (count, keep) or None."""
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top, "scale": scale,
                                      "groups": None if groups is None else dict(zip(("count", "keep"), groups))},
            "expert": {"ff": ff}, "shared": None if shared is None else {"ff": shared}}


def layer(type_, heads, kv_heads, dim, vdim, window=0, rot=None, base=10000.0, scaling=None, scale=0.25, v_mix=True, mlp=None):
    """rot: rotated values per head (None for layers that know no positions); scaling: (factor, original, fast, slow)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if window:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"dims": rot, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": type_, "mixer": m, "mlp": mlp}


def config(layers, vocab=96, width=48, eps=1e-5, embedding_scale=3.0, logit_scale=0.75):
    return {"architecture": "Silevik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_scale": logit_scale,
            "embedding": {"scale": embedding_scale}}


def shapes(cfg):
    d = cfg["width"]
    out = {"embed": (cfg["vocab"], d), "head": (cfg["vocab"], d), "final.norm": (d,), "final.norm.b": (d,)}
    gated = lambda p, f: {p + "gate": (f, d), p + "up": (f, d), p + "down": (d, f)}
    for i, spec in enumerate(cfg["layers"]):
        m, p, kind = spec["mixer"], f"l{i}.", R.KINDS[spec["type"]]
        H, G, k, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if spec["mlp"] else ()):
            out.update({p + n: (d,), p + n + ".b": (d,)})
        out.update({p + "mix.q": (H * k, d), p + "mix.k": (G * k, d), p + "mix.v": (G * v, d), p + "mix.o": (d, H * v)})
        if kind["norm"]:
            out.update({p + "mix.q.norm": (k if kind["norm"] == "head" else H * k,), p + "mix.k.norm": (k if kind["norm"] == "head" else G * k,)})
        if kind["sink"]:
            out[p + "mix.sink"] = (H,)
        if kind["gate"]:
            out[p + "mix.g"] = (H if kind["gate"] == "head" else H * v, d)
        if m["v_mix"]:
            out[p + "mix.vmix"] = ()
        mlp = spec["mlp"]
        if mlp and mlp["kind"] == "dense":
            out.update(gated(p + "mlp.", mlp["ff"]))
        elif mlp:
            n = mlp["router"]["experts"] + mlp["router"]["identity"]
            out.update({p + "mlp.router": (n, d), p + "mlp.correction": (n,)})
            for e in range(mlp["router"]["experts"]):
                out.update(gated(f"{p}mlp.e{e}.", mlp["expert"]["ff"]))
            if mlp["shared"]:
                out.update({**gated(p + "mlp.shared.", mlp["shared"]["ff"]), p + "mlp.shared.sg": (1, d)})
    return out


def random_weights(cfg, seed=0):
    """bf16-representable float32 weights. Scores are sharp, sinks, gates and corrections matter, so that a key on the wrong side of a
    window's edge, a sink left out or a wrong expert moves the logits."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in shapes(cfg).items():
        x = rng.standard_normal(shape)
        if name.endswith(("norm.b", "norm1.b", "norm2.b", "norm1b.b", "norm2b.b")):
            x = 0.3 * x
        elif name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
            x = 1.0 + 0.25 * x
            if name.endswith(("q.norm", "k.norm")):
                x = x * 1.6
        elif name.endswith("sink"):
            x = x + 2.0
        elif name.endswith("vmix"):
            x = rng.uniform(0.2, 0.8, shape)
        elif name.endswith("correction"):
            x = 0.6 * x - 0.5
        elif name not in ("embed",):
            x = x / np.sqrt(shape[-1])
            if name.endswith(("mix.q", "mix.k")):
                x = x * 1.6
            elif name.endswith(("router", "mix.g")):
                x = x * 2.0
        w[name] = M.from_bf16(M.to_bf16(np.asarray(x))).reshape(shape)
    return w


def wide(weights):
    return {k: v.astype(np.float64) for k, v in weights.items()}


def reference_logits(cfg, weights, tokens, residuals=None):
    return R.forward(tokens, wide(weights), cfg, residuals)


def clear_choices(cfg, weights, tokens, gap=0.03):
    """[n] bool: positions at which every router's choice is clear (the best group and the best expert left out are `gap` behind)."""
    W, eps = wide(weights), cfg["norm"]["eps"]
    clear = np.ones(len(tokens), bool)
    x, first = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"], []
    for i, spec in enumerate(cfg["layers"]):
        mlp, p = spec["mlp"], f"l{i}."
        mid = dict(cfg, layers=cfg["layers"][:i] + [dict(spec, mlp=None)])
        after_mixer = R.layer(x, W, i, mid, list(first))
        if mlp and mlp["kind"] == "moe":
            r = mlp["router"]
            z = R.layer_norm(after_mixer, W[p + "norm2"], W[p + "norm2.b"], eps) @ W[p + "mlp.router"].T
            s = np.exp(z - z.max(axis=1, keepdims=True))
            choice = s / s.sum(axis=1, keepdims=True) + W[p + "mlp.correction"]
            g = r["groups"] or {"count": 1, "keep": 1}
            best = choice.reshape(len(tokens), g["count"], -1).max(axis=2)
            order = np.sort(best, axis=1)[:, ::-1]
            if g["keep"] < g["count"]:
                clear &= order[:, g["keep"] - 1] - order[:, g["keep"]] > gap
            choice = np.where(np.repeat(best >= order[:, [g["keep"] - 1]], choice.shape[1] // g["count"], axis=1), choice, -np.inf)
            order = np.sort(choice, axis=1)[:, ::-1]
            if r["top"] < choice.shape[1]:
                clear &= order[:, r["top"] - 1] - order[:, r["top"]] > gap
        x = R.layer(x, W, i, cfg, first)
    return clear
