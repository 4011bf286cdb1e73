"""Plain, slow implementation of the Nigenex decoder in float64, one function per mechanism.

Test infrastructure: nothing of the package is imported here, and the package does not import this.  Weights are a
dict name -> numpy array (any float type, converted to float64), the configuration is the parsed config.json.
"""
import numpy as np


def rms_norm_scalar(x, gain, eps):
    """x / sqrt(mean(x^2) + eps), times one gain shared by all coordinates."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * gain


def token_shift(h, mu, previous=None):
    """Every token's row moves towards the row before it by the fraction mu (per coordinate); `previous` is the row
    before the first one (zeros at the start of a sequence)."""
    prev = np.zeros_like(h)
    prev[1:] = h[:-1]
    if previous is not None:
        prev[0] = previous
    return h + (prev - h) * mu


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def soft_cap(s, cap):
    return cap * np.tanh(s / cap)


def log_distance_bias(r1, r2, distance):
    """What a head subtracts from the score of a key `distance` tokens back."""
    return r1 * np.log(1.0 + r2 * distance)


def window_mask(n_query, n_key, first_query, window):
    """mask[i, j]: the query at position first_query + i sees key j."""
    d = (first_query + np.arange(n_query))[:, None] - np.arange(n_key)[None, :]
    return (d >= 0) & (d < window)


def attention(q, k, v, scale, cap, r1, r2, window, first_query=0):
    """q [n, H, D] at positions first_query .., k / v [m, G, D] at positions 0 ..; returns [n, H, D]."""
    n, H, _ = q.shape
    m, G, _ = k.shape
    out = np.zeros((n, H, v.shape[-1]))
    mask = window_mask(n, m, first_query, window)
    dist = np.maximum((first_query + np.arange(n))[:, None] - np.arange(m)[None, :], 0).astype(np.float64)
    for h in range(H):
        g = h // (H // G)
        s = soft_cap(q[:, h] @ k[:, g].T * scale, cap) - log_distance_bias(r1[h], r2[h], dist)
        s = np.where(mask, s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, g]
    return out


def head_gate(out, logits):
    """Each head's output times the sigmoid of its gate number: out [n, H, D], logits [n, H]."""
    return out * (1.0 / (1.0 + np.exp(-logits)))[:, :, None]


def mixer(w, prefix, cfg, h):
    n = h.shape[0]
    H, G, D = cfg["heads"], cfg["kv_heads"], cfg["dim"]
    q = (h @ w[prefix + "q"].T).reshape(n, H, D)
    k = (h @ w[prefix + "k"].T).reshape(n, G, D)
    o = attention(q, k, k, cfg["scale"], cfg["softcap"], w[prefix + "r1"], w[prefix + "r2"], cfg["mask"]["size"])
    o = head_gate(o, h @ w[prefix + "g"].T)
    return o.reshape(n, H * D) @ w[prefix + "o"].T


def feed_forward(w, prefix, h):
    return (gelu_tanh(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def layer(w, i, cfg, eps, x):
    p = "l%d." % i
    h = rms_norm_scalar(x, w[p + "norm1"], eps)
    y = mixer(w, p + "mix.", cfg["mixer"], token_shift(h, w[p + "shift"]))
    if cfg["mlp"] is not None:
        y = y + feed_forward(w, p + "mlp.", h)
    return x + y


def head(w, cfg, x):
    h = rms_norm_scalar(x, w["final.norm"], cfg["norm"]["eps"])
    return soft_cap(h @ w["head"].T, cfg["logit_softcap"])


def forward(weights, cfg, tokens, collect=None):
    """Logits [n, vocab] of a whole sequence; the residual stream after each layer is appended to `collect`."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    x = w["embed"][np.asarray(tokens)]
    for i, lc in enumerate(cfg["layers"]):
        x = layer(w, i, lc, cfg["norm"]["eps"], x)
        if collect is not None:
            collect.append(x)
    return head(w, cfg, x)
