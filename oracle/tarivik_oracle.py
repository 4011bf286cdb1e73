"""Plain, slow implementation of the Tarivik decoder in float64, one function per mechanism.

Test infrastructure: nothing of the package is imported here, and the package does not import this.  Weights are a
dict name -> numpy array (any float type, converted to float64), the configuration is the parsed config.json.  The recurrent
mixers are written as their recurrences, token by token.
"""
import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def grouped_rms_norm(x, weight, groups, eps):
    """Every group of neighbouring coordinates by its own root mean square, then one weight per coordinate."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return rms(parts, eps).reshape(x.shape) * weight


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def short_conv(h, taps_weight, bias=None):
    """h [n, channels] -> sum over taps of weight[:, j] * h at (t - taps + 1 + j); zeros before the start."""
    taps = taps_weight.shape[1]
    past = np.concatenate([np.zeros((taps - 1, h.shape[1])), h])
    y = sum(taps_weight[:, j] * past[j:j + h.shape[0]] for j in range(taps))
    return y if bias is None else y + bias


def alibi_slopes(heads):
    return 2.0 ** (-8.0 * (np.arange(heads) + 1) / heads)


def chunked_attention(q, k, v, scale, chunk, slopes, sink):
    """q [n, H, D], k [n, G, D], v [n, G, E] of one sequence from its start; a query sees the keys of its own chunk up to itself.
    Scores lose slope * distance; the sink is one more score of the sum."""
    n, H, _ = q.shape
    G = k.shape[1]
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen = (j <= i) & (i // chunk == j // chunk)
    out = np.zeros((n, H, v.shape[-1]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, q[:, h] @ k[:, g].T * scale - slopes[h] * (i - j), -np.inf)
        top = np.maximum(s.max(axis=1, keepdims=True), sink[h])
        p = np.exp(s - top)
        out[:, h] = (p / (p.sum(axis=1, keepdims=True) + np.exp(sink[h] - top))) @ v[:, g]
    return out


def attention(w, p, m, h, eps):
    n = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]
    k = rms(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]
    v = h @ w[p + "v"].T + w[p + "v.b"]
    o = chunked_attention(q.reshape(n, H, D), k.reshape(n, G, D), v.reshape(n, G, E), m["scale"], m["mask"]["size"], alibi_slopes(H), w[p + "sink"])
    return (o.reshape(n, H * E) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def decayed_outer_products(q, k, v, decay, state=None):
    """S_t = diag(decay_t) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t.  q, k, decay [n, H, D], v [n, H, E]; returns o [n, H, E]."""
    n, H, D = q.shape
    S = np.zeros((H, D, v.shape[-1])) if state is None else state.copy()
    out = np.zeros(v.shape)
    for t in range(n):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", S, q[t])
    return out


def hgrn2(w, p, m, h, eps):
    n, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(n, H, D)
    v = (h @ w[p + "v"].T).reshape(n, H, E)
    low = w[p + "lower"]
    f = (low + (1.0 - low) * sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).reshape(n, H, D)
    o = decayed_outer_products(q, 1.0 - f, v, f)
    return (rms(o, eps) * w[p + "norm"]).reshape(n, H * E) @ w[p + "o"].T


def mlstm(w, p, m, h, eps):
    n, H, D, E, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).reshape(n, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).reshape(n, H, D)
    v = (h @ w[p + "v"].T).reshape(n, H, E)
    i = cap * np.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    S, norm, top = np.zeros((H, D, E)), np.zeros((H, D)), np.zeros(H)
    o = np.zeros((n, H, E))
    for t in range(n):
        new = np.maximum(f[t] + top, i[t])
        keep, write = np.exp(f[t] + top - new), np.exp(i[t] - new)
        top = new
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        norm = keep[:, None] * norm + write[:, None] * k[t]
        o[t] = np.einsum("hde,hd->he", S, q[t]) / (np.maximum(np.abs(np.sum(norm * q[t], axis=1)), np.exp(-top)) + 1e-6)[:, None]
    y = rms(o, eps).reshape(n, H * E) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


def mamba2(w, p, m, h, eps):
    n, H, E, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * E
    y = h @ w[p + "in"].T
    z, mixed, dt = y[:, :inner], y[:, inner:2 * inner + 2 * G * N], y[:, 2 * inner + 2 * G * N:]
    mixed = silu(short_conv(mixed, w[p + "conv"], w[p + "conv.b"]))
    x = mixed[:, :inner].reshape(n, H, E)
    B = np.repeat(mixed[:, inner:inner + G * N].reshape(n, G, N), H // G, axis=1)
    C = np.repeat(mixed[:, inner + G * N:].reshape(n, G, N), H // G, axis=1)
    dt = softplus(dt + w[p + "dt_bias"])
    decay = np.exp(-np.exp(w[p + "A_log"]) * dt)
    o = decayed_outer_products(C, B * dt[:, :, None], x, np.broadcast_to(decay[:, :, None], B.shape)) + w[p + "D"][:, None] * x
    return grouped_rms_norm(o.reshape(n, inner) * silu(z), w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


def mixer(w, p, kind, m, h, eps):
    if kind == "parallel":
        return m["left_scale"] * attention(w, p + "left.", m["left"], h, eps) + m["right_scale"] * mamba2(w, p + "right.", m["right"], h, eps)
    return {"hgrn2": hgrn2, "mlstm": mlstm}[kind](w, p, m, h, eps)


def choose_experts(scores, correction, groups, keep, top):
    """Indices [n, top] of the largest corrected scores inside the best groups (a group's worth: its two largest)."""
    n, E = scores.shape
    choice = scores + correction
    parts = choice.reshape(n, groups, E // groups)
    worth = np.sort(parts, axis=-1)[..., -2:].sum(axis=-1)
    best = np.argsort(-worth, axis=-1, kind="stable")[:, :keep]
    allowed = np.zeros((n, groups), dtype=bool)
    np.put_along_axis(allowed, best, True, axis=-1)
    choice = np.where(np.repeat(allowed, E // groups, axis=1), choice, -np.inf)
    return np.argsort(-choice, axis=-1, kind="stable")[:, :top]


def mixture(w, p, m, h):
    r = m["router"]
    scores = sigmoid(h @ w[p + "router"].T)
    chosen = choose_experts(scores, w[p + "correction"], r["groups"]["count"], r["groups"]["keep"], r["top"])
    y = np.zeros_like(h)
    for e in range(r["experts"]):
        t, _ = np.nonzero(chosen == e)
        q = p + "e%d." % e
        y[t] += scores[t, e][:, None] * ((silu(h[t] @ w[q + "gate"].T) * (h[t] @ w[q + "up"].T)) @ w[q + "down"].T)
    return y


def layer(w, i, cfg, x):
    lc, p = cfg["layers"][i], "l%d." % i
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    h = x + short_conv(x, w[p + "canon1"])
    x = x + grouped_rms_norm(mixer(w, p + "mix.", lc["type"], lc["mixer"], h, eps), w[p + "norm1"], groups, eps)
    if lc["mlp"] is not None:
        h = x + short_conv(x, w[p + "canon2"])
        x = x + grouped_rms_norm(mixture(w, p + "mlp.", lc["mlp"], h), w[p + "norm2"], groups, eps)
    return x


def forward(weights, cfg, tokens, collect=None):
    """Logits [n, vocab] of a whole sequence; the residual stream after each layer is appended to `collect`."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    x = w["embed"][np.asarray(tokens)] + w["pos"][:len(tokens)]
    for i in range(len(cfg["layers"])):
        x = layer(w, i, cfg, x)
        if collect is not None:
            collect.append(x)
    return grouped_rms_norm(x, w["final.norm"], cfg["norm"]["groups"], cfg["norm"]["eps"]) @ w["head"].T
