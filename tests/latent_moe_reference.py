"""Plain NumPy statement of the looped latent-attention / mixture-of-experts decoder ("Banevik"): what the CUDA path is tested against.

The slow textbook form in float64 (or whatever dtype the weights have): one function per mechanism, loops over tokens, heads and
experts, no code shared with the product. A model is a dict of weights (name -> ndarray) and the parsed config.json.
"""
import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1.0 + w)


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Table row of every token, hashed from the pair it ends; the row behind the hashed ones stands for having no predecessor."""
    rows = [buckets]
    for a, b in zip(tokens[:-1], tokens[1:]):
        rows.append((int(a) * mul_prev + int(b) * mul_cur) % buckets)
    return np.array(rows[:len(tokens)])


def embed(tokens, W, cfg):
    x = W["embed"][np.asarray(tokens)].copy()
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram:
        x = x + W["bigram"][bigram_rows(tokens, bigram["buckets"], bigram["mul_prev"], bigram["mul_cur"])]
    return x


def rotate(x, positions, dims, base):
    """Rotates the first `dims` values of the last axis of x [n, ..., d]: value i with value i + dims / 2, by p * base^(-2 i / dims)."""
    half = dims // 2
    out = x.copy()
    for t, p in enumerate(positions):
        for i in range(half):
            a = p * float(base) ** (-2.0 * i / dims)
            u, v = x[t, ..., i].copy(), x[t, ..., i + half].copy()
            out[t, ..., i] = u * np.cos(a) - v * np.sin(a)
            out[t, ..., i + half] = v * np.cos(a) + u * np.sin(a)
    return out


def window_visible(n, size):
    """[n, n] bool: query i sees keys i - size + 1 .. i (size 0: 0 .. i)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (size == 0))


def softmax_with_sink(s, sink):
    """Rows of exp(s) over their sum plus exp(sink); -inf entries are not seen."""
    m = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def latent(h, W, p, m, eps):
    """(c [n, rank] normalised, rotated key part [n, rot_dim]): all that a cache has to hold."""
    d = h @ W[p + "dkv"].T
    c = rms(d[:, :m["kv_rank"]], eps) * W[p + "dkv.norm"]
    return c, rotate(d[:, m["kv_rank"]:], np.arange(h.shape[0]), m["rot"]["dims"], m["rot"]["base"])


def latent_attention(h, W, p, m, eps):
    n, H, d, r, v = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ W[p + "q"].T).reshape(n, H, d + r)
    qr = rotate(q[:, :, d:], np.arange(n), m["rot"]["dims"], m["rot"]["base"])
    c, kr = latent(h, W, p, m, eps)
    k = (c @ W[p + "uk"].T).reshape(n, H, d)
    val = (c @ W[p + "uv"].T).reshape(n, H, v)
    see = window_visible(n, m["mask"]["size"] if m.get("mask") else 0)
    out = np.zeros((n, H, v), dtype=h.dtype)
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        out[:, i] = softmax_with_sink(np.where(see, s, -np.inf), W[p + "sink"][i]) @ val[:, i]
    return out.reshape(n, H * v) @ W[p + "o"].T


def route(h, w_router, top):
    """(experts [n, top], weights [n, top]): the top sigmoid scores, larger first; nothing is normalised."""
    s = 1.0 / (1.0 + np.exp(-(h @ w_router.T)))
    best = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return best, np.take_along_axis(s, best, axis=1)


def expert(z, up, down):
    return np.square(np.maximum(z @ up.T, 0.0)) @ down.T


def mixture(h, W, p, m):
    best, s = route(h, W[p + "router"], m["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(best[t], s[t]):
            out[t] += expert(w * h[t], W[f"{p}e{e}.up"], W[f"{p}e{e}.down"])
    return out


def layer(x, W, p, cfg, i, eps):
    spec = cfg["layers"][i]
    if spec["type"] != "latent_attention":
        raise ValueError(spec["type"])
    y = latent_attention(offset_norm(x, W[p + "norm1"], eps), W, p + "mix.", spec["mixer"], eps)
    if spec.get("mlp"):
        y = y + mixture(offset_norm(x, W[p + "norm2"], eps), W, p + "mlp.", spec["mlp"])
    return x + y


def layer_runs(cfg):
    """[(layer, first of a pass)] in the order of execution."""
    loop, out, i = cfg.get("loop"), [], 0
    while i < len(cfg["layers"]):
        if loop and i == loop["start"]:
            for _ in range(loop["times"]):
                out += [(j, j == loop["start"]) for j in range(loop["start"], loop["stop"])]
            i = loop["stop"]
        else:
            out.append((i, False))
            i += 1
    return out


def forward(tokens, W, cfg, residuals=None):
    """Logits [n, vocab] of a whole sequence; `residuals` (a list) receives the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = embed(tokens, W, cfg)
    x = x0
    for i, entry in layer_runs(cfg):
        if entry:
            x = np.concatenate([x, x0], axis=1) @ W["loop.in"].T
        x = layer(x, W, f"l{i}.", cfg, i, eps)
        if residuals is not None:
            residuals.append(x.copy())
    logits = offset_norm(x, W["final.norm"], eps) @ W["embed"].T
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(logits / cap) if cap else logits
