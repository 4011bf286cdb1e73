"""Plain, slow implementation of the Gimozen decoder in float64, one function per mechanism.

Test infrastructure: nothing of the package is imported here, and the package does not import this.  Weights are a
dict name -> numpy array (any float type, converted to float64), the configuration is the parsed config.json.
"""
import math

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def rms_norm_zero_centred(x, weight, eps):
    """The stored weight is the distance from one."""
    return rms(x, eps) * (1.0 + weight)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rotary_frequencies(dims, base, scaling=None):
    """Radians per position of the dims / 2 rotated pairs; scaling: frequencies blended between f and f / factor by how
    often a pair turns within the original context."""
    i = np.arange(dims // 2, dtype=np.float64)
    f = base ** (-2.0 * i / dims)
    if scaling is None:
        return f

    def pair_with_turns(t):
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo = max(math.floor(pair_with_turns(scaling["fast"])), 0)
    hi = min(math.ceil(pair_with_turns(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp)


def rotary_magnitude(scaling=None):
    return 1.0 if scaling is None else 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [n, ..., D]: the first rot['dims'] columns in half-split pairs, the others unchanged."""
    dims, scaling = rot["dims"], rot.get("scaling")
    a = np.asarray(positions, dtype=np.float64)[:, None] * rotary_frequencies(dims, rot["base"], scaling)
    m = rotary_magnitude(scaling)
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (dims // 2,)
    c, s = (m * np.cos(a)).reshape(shape), (m * np.sin(a)).reshape(shape)
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions, dtype=np.float64) + 1) / every) + 1.0)


def causal_attention(q, k, v, scale, sink=None, first_query=0):
    """q [n, H, D] at positions first_query .., k [m, G, D] and v [m, G, E] at positions 0 ..; returns [n, H, E].
    sink [H]: one more score per head that weighs in the sum and has no value."""
    n, H, _ = q.shape
    m, G, _ = k.shape
    seen = (first_query + np.arange(n))[:, None] >= np.arange(m)[None, :]
    out = np.zeros((n, H, v.shape[-1]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, q[:, h] @ k[:, g].T * scale, -np.inf)
        top = s.max(axis=1, keepdims=True)
        if sink is not None:
            top = np.maximum(top, sink[h])
        p = np.exp(s - top)
        total = p.sum(axis=1, keepdims=True)
        if sink is not None:
            total = total + np.exp(sink[h] - top)
        out[:, h] = (p / total) @ v[:, g]
    return out


def latent_of(w, prefix, m, h, eps):
    """What a latent layer caches of the rows h: the normed latents [n, kv_rank] and the rotated key part [n, rot_dim]."""
    y = h @ w[prefix + "dkv"].T
    r = m["kv_rank"]
    return rms_norm(y[:, :r], w[prefix + "dkv.norm"], eps), rotate(y[:, r:], np.arange(h.shape[0]), m["rot"])


def latent_attention(w, prefix, m, h, latent):
    n = h.shape[0]
    H, D, R, E = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, key_rot = latent
    q = (h @ w[prefix + "q"].T).reshape(n, H, D + R)
    q = np.concatenate([q[..., :D], rotate(q[..., D:], np.arange(n), m["rot"])], axis=-1)
    k = np.concatenate([(c @ w[prefix + "uk"].T).reshape(n, H, D), np.broadcast_to(key_rot[:, None], (n, H, R))], axis=-1)
    v = (c @ w[prefix + "uv"].T).reshape(n, H, E)
    o = causal_attention(q, k, v, m["scale"], w[prefix + "sink"]).reshape(n, H * E)
    return (o * sigmoid(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def attention(w, prefix, m, h, eps):
    n = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w[prefix + "q"].T).reshape(n, H, D), w[prefix + "q.norm"], eps)
    k = rms_norm((h @ w[prefix + "k"].T).reshape(n, G, D), w[prefix + "k.norm"], eps)
    v = (h @ w[prefix + "v"].T).reshape(n, G, E)
    t = m.get("q_temp")
    if t is not None:
        q = q * query_temperature(np.arange(n), t["coef"], t["every"])[:, None, None]
    return causal_attention(q, k, v, m["scale"]).reshape(n, H * E) @ w[prefix + "o"].T


def feed_forward(w, prefix, h):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def layer(w, i, cfg, x, latents):
    """latents: per layer what it caches; layers that borrow read it here."""
    lc, eps, alpha, p = cfg["layers"][i], cfg["norm"]["eps"], cfg["postln_alpha"], "l%d." % i
    m = lc["mixer"]
    if lc["type"] == "latent_attention":
        source = m.get("kv_from")
        if source is None:
            latents[i] = latent_of(w, p + "mix.", m, x, eps)
        y = latent_attention(w, p + "mix.", m, x, latents[i if source is None else source])
    else:
        y = attention(w, p + "mix.", m, x, eps)
    x = rms_norm_zero_centred(alpha * x + y, w[p + "norm1"], eps)
    if lc["mlp"] is not None:
        x = rms_norm_zero_centred(alpha * x + feed_forward(w, p + "mlp.", x), w[p + "norm2"], eps)
    return x


def forward(weights, cfg, tokens, collect=None):
    """Logits [n, vocab] of a whole sequence; the residual stream after each layer is appended to `collect`."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    latents = {}
    for i in range(len(cfg["layers"])):
        x = layer(w, i, cfg, x, latents)
        if collect is not None:
            collect.append(x)
    return rms_norm_zero_centred(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
