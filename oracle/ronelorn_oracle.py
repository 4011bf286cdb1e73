"""Plain, slow implementation of the Ronelorn decoder in float64, one function per mechanism.

Test infrastructure: nothing of the package is imported here, and the package does not import this.  Weights are a
dict name -> numpy array (any float type, converted to float64), the configuration is the parsed config.json.  Visibility is
written as its definition, key by key; the recurrence token by token.
"""
import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def shifted_rms_norm(x, w, eps):
    """The weight is stored as its distance from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def frequencies(base, dims, factor=None):
    f = base ** (-2.0 * np.arange(dims // 2) / dims)
    return f if factor is None else f / factor


def rotate_half(x, positions, freq):
    """x [n, heads, D]: coordinates i and i + len(freq) turn by positions * freq[i]; the rest pass."""
    half = len(freq)
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * freq
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., 2 * half:]], axis=-1)


def softcap(s, cap):
    return cap * np.tanh(s / cap)


def window_mask(n, size):
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & (i - j < size)


def kept_mask(n, size, keep):
    """The window, and the first `keep` tokens for good."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep))


def block_mask(n, size, pool):
    """[n, whole blocks]: block b, of the positions b pool .. b pool + pool - 1, lies wholly before the window of row i."""
    i, b = np.arange(n)[:, None], np.arange(n // pool)[None, :]
    return b * pool + pool - 1 <= i - size


def block_means(x, pool):
    """x [n, heads, D] -> means over whole blocks of `pool` rows."""
    whole = x.shape[0] // pool
    return x[:whole * pool].reshape((whole, pool) + x.shape[1:]).mean(axis=1)


def softmax_sum(scores, seen, values, one_more):
    """Sum of values [m, E] by the softmax of scores [n, m] where seen; one_more: a score of zero without a value joins the sum."""
    s = np.where(seen, scores, -np.inf)
    top = s.max(axis=1, keepdims=True)
    if one_more:
        top = np.maximum(top, 0.0)
    p = np.exp(s - top)
    return (p / (p.sum(axis=1, keepdims=True) + (np.exp(-top) if one_more else 0.0))) @ values


def grouped_attention(q, k, v, seen, scale, cap=None, one_more=False):
    """q [n, H, D], k [m, G, D], v [m, G, E], seen [n, m] -> [n, H, E]."""
    H, G = q.shape[1], k.shape[1]
    out = np.zeros((q.shape[0], H, v.shape[-1]))
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        out[:, h] = softmax_sum(s if cap is None else softcap(s, cap), seen, v[:, g], one_more)
    return out


def pooled_window_attention(w, p, m, h, eps):
    """Norms per head, scaled rotation of queries and keys, values that turn with their position, capped scores; tokens of the window
    beside means of the blocks before it."""
    n, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, rot = np.arange(n), m["rot"]
    f = frequencies(rot["base"], rot["dims"], (rot.get("scaling") or {}).get("factor"))
    q = rotate_half(rms((h @ w[p + "q"].T).reshape(n, H, D), eps) * w[p + "q.norm"], pos, f)
    k = rotate_half(rms((h @ w[p + "k"].T).reshape(n, G, D), eps) * w[p + "k.norm"], pos, f)
    turn = frequencies(rot["base"], E)
    v = rotate_half((h @ w[p + "v"].T).reshape(n, G, E), pos, turn)
    size, pool = m["mask"]["size"], m["mask"]["pool"]
    keys, values = np.concatenate([block_means(k, pool), k]), np.concatenate([block_means(v, pool), v])
    seen = np.concatenate([block_mask(n, size, pool), window_mask(n, size)], axis=1)
    o = rotate_half(grouped_attention(q, keys, values, seen, m["scale"], cap=m["softcap"]), -pos, turn)
    return o.reshape(n, H * E) @ w[p + "o"].T


def kept_window_attention(w, p, m, h, eps):
    """Norms of whole projections, rotation of queries and keys, a sink of score zero; tokens of the window beside the first ones."""
    n, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    f = frequencies(m["rot"]["base"], m["rot"]["dims"], (m["rot"].get("scaling") or {}).get("factor"))
    q = rotate_half((rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).reshape(n, H, D), np.arange(n), f)
    k = rotate_half((rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).reshape(n, G, D), np.arange(n), f)
    v = (h @ w[p + "v"].T).reshape(n, G, E)
    o = grouped_attention(q, k, v, kept_mask(n, m["mask"]["size"], m["mask"]["keep_first"]), m["scale"], one_more=True)
    return o.reshape(n, H * E) @ w[p + "o"].T


def gated_scan(z, candidate, state=None):
    """S_t = (1 - z_t) S_(t-1) + z_t candidate_t, element by element; returns every S_t."""
    S = np.zeros(z.shape[1]) if state is None else np.asarray(state, dtype=np.float64)
    out = np.zeros(z.shape)
    for t in range(z.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * candidate[t]
        out[t] = S
    return out


def positive(u):
    """u + 1/2 from zero on, sigmoid(u) below."""
    return np.where(u >= 0, u + 0.5, sigmoid(u))


def mingru(w, p, m, h, eps):
    z = sigmoid(h @ w[p + "z"].T + w[p + "z.b"])
    s = gated_scan(z, positive(h @ w[p + "x"].T + w[p + "x.b"]))
    return (s * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"attention": pooled_window_attention, "attention_2": kept_window_attention, "mingru": mingru}


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def layer(w, i, cfg, x):
    lc, p, eps, mult = cfg["layers"][i], "l%d." % owner(cfg, i), cfg["norm"]["eps"], cfg["residual_mult"]
    x = x + mult * MIXERS[lc["type"]](w, p + "mix.", lc["mixer"], shifted_rms_norm(x, w[p + "norm1"], eps), eps)
    if lc["mlp"] is not None:
        h = shifted_rms_norm(x, w[p + "norm2"], eps)
        x = x + mult * (squared_relu(h @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T)
    return x


def forward(weights, cfg, tokens, collect=None):
    """Logits [n, vocab] of a whole sequence; the residual stream after each layer is appended to `collect`."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i in range(len(cfg["layers"])):
        x = layer(w, i, cfg, x)
        if collect is not None:
            collect.append(x)
    return shifted_rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
