"""Plain NumPy statement of the hybrid recurrent/attention decoder ("Besudra"), used as the checker of the CUDA path.

Everything here is the slow textbook form in float64 (or whatever dtype is passed): loops over tokens, one function per
mechanism, no code shared with the product. A model is a dict of weights (name -> ndarray) and the parsed config.json.
"""
import numpy as np


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def causal_conv(x, w, b):
    """Per-channel causal convolution: y[t, c] = b[c] + sum_j w[c, j] x[t - (taps - 1) + j, c], zeros before t = 0."""
    n, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x)
    for t in range(n):
        y[t] = b
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] = y[t] + w[:, j] * x[s]
    return y


def chunk_visible(n, size):
    """[n, n] bool: key j is visible to query i (causal, same chunk of `size` positions counted from position 0)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & (i // size == j // size)


def attend(q, k, v, scale, visible):
    """q [n, H, d], k [n, G, d], v [n, G, dv]; query head h reads kv head h // (H / G). Softmax over visible keys."""
    n, n_head, _ = q.shape
    group = n_head // k.shape[1]
    out = np.zeros((n, n_head, v.shape[2]), dtype=q.dtype)
    for h in range(n_head):
        s = (q[:, h] @ k[:, h // group].T) * scale
        s = np.where(visible, s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h // group]
    return out


def chunked_attention(h, W, p, cfg, eps):
    """Attention whose values are the un-normalised keys; q and k normalised over the whole projection; no positions."""
    n, dim = h.shape[0], cfg["dim"]
    q = h @ W[p + "q"].T
    kv = h @ W[p + "k"].T
    qn = rms_norm(q, W[p + "q.norm"], eps).reshape(n, cfg["heads"], dim)
    kn = rms_norm(kv, W[p + "k.norm"], eps).reshape(n, cfg["kv_heads"], dim)
    v = kv.reshape(n, cfg["kv_heads"], dim)
    o = attend(qn, kn, v, cfg["scale"], chunk_visible(n, cfg["mask"]["size"]))
    return o.reshape(n, -1) @ W[p + "o"].T


def block_linear(u, w, b):
    """Block-diagonal product: u [n, blocks * m], w [blocks, m, m] as [out, in], b [blocks, m]."""
    blocks, m, _ = w.shape
    parts = u.reshape(u.shape[0], blocks, m)
    return (np.einsum("nbi,boi->nbo", parts, w) + b).reshape(u.shape[0], -1)


def gated_lru_scan(u, r, i, lam, s0=None):
    """s_t = a_t s_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a_t = -8 r_t softplus(lam). Returns all s_t."""
    s = np.zeros(u.shape[1], dtype=u.dtype) if s0 is None else s0.copy()
    out = np.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        s = np.exp(log_a) * s + np.sqrt(-np.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = s
    return out


def gated_lru_block(h, W, p, cfg):
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = causal_conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    r = sigmoid(block_linear(u, W[p + "ra"], W[p + "ra.b"]))
    i = sigmoid(block_linear(u, W[p + "ri"], W[p + "ri.b"]))
    return (gated_lru_scan(u, r, i, W[p + "lam"]) * y) @ W[p + "o"].T


def parallel_mixer(h, W, p, cfg, eps):
    return (cfg["left_scale"] * chunked_attention(h, W, p + "left.", cfg["left"], eps)
            + cfg["right_scale"] * gated_lru_block(h, W, p + "right.", cfg["right"]))


def selective_scan(x, dt, A, B, C, D, s0=None):
    """x, dt [n, inner], A [inner, N], B, C [n, N], D [inner]: S <- exp(dt A) S + dt x B, y = S C + D x."""
    s = np.zeros_like(A) if s0 is None else s0.copy()
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        s = np.exp(dt[t][:, None] * A) * s + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = s @ C[t] + D * x[t]
    return y


def mamba1_mixer(h, W, p, cfg):
    inner, n_state, rank = cfg["inner"], cfg["state"], cfg["dt_rank"]
    xz = h @ W[p + "in"].T
    x = silu(causal_conv(xz[:, :inner], W[p + "conv"], W[p + "conv.b"]))
    z = xz[:, inner:]
    dbc = x @ W[p + "x"].T
    dt = softplus(dbc[:, :rank] @ W[p + "dt"].T + W[p + "dt.b"])
    B, C = dbc[:, rank:rank + n_state], dbc[:, rank + n_state:]
    y = selective_scan(x, dt, -np.exp(W[p + "A_log"]), B, C, W[p + "D"])
    return (y * silu(z)) @ W[p + "o"].T


def gated_mlp(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def forward(tokens, W, cfg, residuals=None):
    """Logits [n, vocab] of a whole sequence; `residuals` (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)].copy()
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_norm(x, W[p + "norm1"], eps)
        if layer["type"] == "mamba1":
            x = x + mamba1_mixer(h, W, p + "mix.", layer["mixer"])
        elif layer["type"] == "parallel":
            x = x + parallel_mixer(h, W, p + "mix.", layer["mixer"], eps)
        else:
            raise ValueError(layer["type"])
        if layer["mlp"] is not None:
            x = x + gated_mlp(rms_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
        if residuals is not None:
            residuals.append(x.copy())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T
