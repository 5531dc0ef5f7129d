"""Plain NumPy statement of the sandwich-normed attention / grouped-mixture decoder ("Silevik"): what the CUDA path is tested against.

The slow textbook form in float64 (or whatever dtype the weights have): one function per mechanism, loops over tokens, heads and
experts, no code shared with the product. A model is a dict of weights (name -> ndarray) and the parsed config.json.
"""
import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def layer_norm(x, w, b, eps):
    c = x - x.mean(axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(np.square(c), axis=-1, keepdims=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps) * w


def frequencies(dims, base, scaling=None):
    """(radians per position [dims / 2], factor of cosine and sine). Scaled: fast pairs keep their frequency, slow ones are stretched by
    `factor`, those between the pairs that turn `fast` and `slow` times within `original` positions are blended."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return np.array(f), 1.0
    s, n = scaling["factor"], scaling["original"]
    turning = lambda t: dims * np.log(n / (2 * np.pi * t)) / (2 * np.log(float(base)))
    lo = max(np.floor(turning(scaling["fast"])), 0)
    hi = min(np.ceil(turning(scaling["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        stretched = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / s * stretched + v * (1 - stretched))
    return np.array(out), 0.1 * np.log(s) + 1.0


def rotate(x, positions, dims, base, scaling=None):
    """x [n, heads, d]: values 2 i and 2 i + 1 of the first `dims` of every head are turned by position * frequency i."""
    f, gain = frequencies(dims, base, scaling)
    out = x.copy()
    for t, p in enumerate(positions):
        for i in range(dims // 2):
            c, s = gain * np.cos(p * f[i]), gain * np.sin(p * f[i])
            u, v = x[t, :, 2 * i].copy(), x[t, :, 2 * i + 1].copy()
            out[t, :, 2 * i] = u * c - v * s
            out[t, :, 2 * i + 1] = v * c + u * s
    return out


def visible(n, window):
    """[n, n] bool: query i sees keys i - window + 1 .. i (window 0: 0 .. i)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i - j < window) | (window == 0))


def softmax(s, sink=None):
    """Rows of exp(s) over their sum, plus exp(sink) if there is one; -inf entries are not seen."""
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    total = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - m)
    return e / total


def attend(q, k, v, scale, window=0, sink=None):
    """q [n, H, d], k [n, G, d], v [n, G, c] -> [n, H, c]."""
    n, heads, groups = q.shape[0], q.shape[1], k.shape[1]
    see = visible(n, window)
    out = np.zeros((n, heads, v.shape[2]), dtype=q.dtype)
    for h in range(heads):
        g = h // (heads // groups)
        s = np.where(see, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        out[:, h] = softmax(s, None if sink is None else sink[h]) @ v[:, g]
    return out


# What the three kinds of attention layer do besides the common part: where the norm of queries and keys is taken, whether they are
# rotated, whether a head has a sink, and how the result is gated.
KINDS = {
    "attention": {"norm": None, "rotates": True, "sink": False, "gate": "element"},
    "attention_2": {"norm": "head", "rotates": False, "sink": False, "gate": "head"},
    "attention_3": {"norm": "whole", "rotates": True, "sink": True, "gate": None},
}


def queries_keys(h, W, p, kind, m, eps):
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ W[p + "q"].T, h @ W[p + "k"].T
    if kind["norm"] == "whole":
        q, k = rms_norm(q, W[p + "q.norm"], eps), rms_norm(k, W[p + "k.norm"], eps)
    q, k = q.reshape(n, H, d), k.reshape(n, G, d)
    if kind["norm"] == "head":
        q, k = rms_norm(q, W[p + "q.norm"], eps), rms_norm(k, W[p + "k.norm"], eps)
    if kind["rotates"]:
        r = m["rot"]
        q, k = (rotate(x, np.arange(n), r["dims"], r["base"], r.get("scaling")) for x in (q, k))
    return q, k


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def attention(h, W, p, type_, m, eps, first_values):
    """first_values: a list that is empty until the first layer that mixes values has run, and then holds its values."""
    kind, n = KINDS[type_], h.shape[0]
    q, k = queries_keys(h, W, p, kind, m, eps)
    v = (h @ W[p + "v"].T).reshape(n, m["kv_heads"], m["vdim"])
    if m.get("v_mix"):
        if first_values:
            v = mix_values(v, first_values[0], W[p + "vmix"])
        else:
            first_values.append(v)
    y = attend(q, k, v, m["scale"], m["mask"]["size"] if m.get("mask") else 0, W[p + "sink"] if kind["sink"] else None)
    if kind["gate"] == "head":
        y = y * sigmoid(h @ W[p + "g"].T)[:, :, None]
    y = y.reshape(n, -1)
    if kind["gate"] == "element":
        y = y * sigmoid(h @ W[p + "g"].T)
    return y @ W[p + "o"].T


def gated_mlp(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, w_router, correction, top, count, keep, scale):
    """(chosen [n, top], weights [n, top]), larger choice score first. Only choices of the `keep` best of `count` groups of neighbours
    stand; a group is as good as its best choice."""
    z = h @ w_router.T
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = s / s.sum(axis=1, keepdims=True)
    choice = s + correction
    n, per = z.shape[1], z.shape[1] // count
    chosen = np.zeros((len(h), top), int)
    for t in range(len(h)):
        groups = sorted(range(count), key=lambda g: -choice[t, g * per:(g + 1) * per].max())[:keep]
        open_ = [e for e in range(n) if e // per in groups]
        chosen[t] = sorted(open_, key=lambda e: -choice[t, e])[:top]
    w = np.take_along_axis(s, chosen, axis=1)
    return chosen, w / (w.sum(axis=1, keepdims=True) + 1e-20) * scale


def mixture(h, W, p, mlp):
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    chosen, weight = route(h, W[p + "router"], W[p + "correction"], r["top"], groups["count"], groups["keep"], r["scale"])
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, w in zip(chosen[t], weight[t]):
            out[t] += w * (h[t] if e >= r["experts"] else gated_mlp(h[t], W, f"{p}e{e}."))
    if mlp.get("shared"):
        out = out + sigmoid(h @ W[p + "shared.sg"].T) * gated_mlp(h, W, p + "shared.")
    return out


def layer(x, W, i, cfg, first_values):
    spec, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    norm = lambda v, name: layer_norm(v, W[p + name], W[p + name + ".b"], eps)
    x = x + norm(attention(norm(x, "norm1"), W, p + "mix.", spec["type"], spec["mixer"], eps, first_values), "norm1b")
    if spec.get("mlp"):
        h = norm(x, "norm2")
        x = x + norm(gated_mlp(h, W, p + "mlp.") if spec["mlp"]["kind"] == "dense" else mixture(h, W, p + "mlp.", spec["mlp"]), "norm2b")
    return x


def forward(tokens, W, cfg, residuals=None):
    """Logits [n, vocab] of a whole sequence; `residuals` (a list) receives the residual stream after every layer."""
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    first_values = []
    for i in range(len(cfg["layers"])):
        x = layer(x, W, i, cfg, first_values)
        if residuals is not None:
            residuals.append(x.copy())
    return layer_norm(x, W["final.norm"], W["final.norm.b"], cfg["norm"]["eps"]) @ W["head"].T * cfg["logit_scale"]
