"""Small random Tarivik models for the tests: configurations, weights, model folders."""
import numpy as np

from oracle import tarivik_oracle as to
from tests.nigenex_models import logit_error, write_folder  # noqa: F401  (shared by the tests of the designs)
from turbospark_b200.plain import bf16_bits, bf16_to_f32


def moe(ff, experts, top, groups, keep):
    return None if ff is None else {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


def parallel(left, right, mlp, scales=(0.8, 1.1), scale=None):
    """left: heads, kv_heads, dim, vdim, chunk; right: heads, groups, vdim, state, conv, norm_groups."""
    H, G, D, E, chunk = left
    h, g, v, n, conv, ng = right
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": H, "kv_heads": G, "dim": D, "vdim": E, "mask": {"size": chunk}, "scale": 1.3 / D ** 0.5 if scale is None else scale},
        "right": {"heads": h, "groups": g, "vdim": v, "state": n, "conv": conv, "norm_groups": ng}, "left_scale": scales[0], "right_scale": scales[1]}}


def hgrn2(heads, dim, vdim, mlp):
    return {"type": "hgrn2", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def mlstm(heads, dim, vdim, mlp, cap=9.0):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def config(width, vocab, layers, groups=2, taps=3, eps=1e-5, positions=640):
    return {"architecture": "Tarivik", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups}, "canon": {"taps": taps}, "max_positions": positions,
            "layers": layers}


# name -> configuration.  Sizes that divide nothing evenly, sizes that happen to be equal or one, layers that differ.
CONFIGS = {
    "odd": config(200, 333, [parallel((6, 3, 40, 24, 37), (6, 3, 20, 24, 4, 2), moe(40, 10, 3, 5, 2)), hgrn2(5, 24, 33, moe(24, 6, 2, 2, 1)),
                             mlstm(3, 20, 28, moe(40, 10, 3, 5, 2)), parallel((4, 2, 20, 28, 100), (3, 1, 16, 8, 2, 3), None)], groups=5, eps=1e-3),
    # whole vectors and tensor tiles everywhere
    "even": config(256, 130, [mlstm(2, 128, 64, moe(64, 16, 4, 4, 2)), parallel((8, 1, 64, 64, 64), (4, 1, 64, 128, 4, 1), moe(64, 16, 4, 4, 2)),
                              hgrn2(2, 128, 64, moe(128, 8, 2, 2, 2)), hgrn2(4, 64, 96, None)], taps=4),
    # heads that no tensor kernel takes, many taps
    "large": config(96, 64, [hgrn2(2, 136, 40, None), mlstm(1, 260, 72, moe(16, 4, 1, 1, 1)), parallel((2, 1, 160, 130, 90), (2, 2, 72, 200, 7, 4), None)], groups=3, taps=6),
    # more experts than are ranked at once; a chunk that no prompt of the tests leaves
    "many_experts": config(128, 75, [parallel((4, 4, 16, 16, 1000), (8, 4, 16, 16, 4, 8), moe(8, 130, 5, 13, 4)), mlstm(4, 16, 8, moe(8, 64, 8, 8, 3))], groups=4),
    # constants and sizes that are one
    "ones": config(64, 40, [parallel((1, 1, 16, 8, 1), (1, 1, 8, 8, 1, 1), moe(8, 1, 1, 1, 1), scales=(1.0, 1.0)), hgrn2(1, 8, 8, moe(8, 3, 3, 3, 3)),
                            mlstm(1, 8, 8, None, cap=1.0)], groups=1, taps=1),
}


def rounded(w):
    return {k: bf16_to_f32(bf16_bits(v)).reshape(np.shape(v)) for k, v in w.items()}


def random_weights(cfg, seed):
    """name -> float32 array whose values are bfloat16 numbers."""
    rng = np.random.default_rng(seed)
    d, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]

    def mat(rows, cols, gain=1.0):
        return rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    w = {"embed": rng.standard_normal((V, d)) * 0.8, "pos": rng.standard_normal((cfg["max_positions"], d)) * 0.3, "head": mat(V, d, 2.0),
         "final.norm": rng.uniform(0.6, 1.4, d)}
    for i, l in enumerate(cfg["layers"]):
        p, m = "l%d." % i, l["mixer"]
        q = p + "mix."
        w[p + "norm1"], w[p + "canon1"] = rng.uniform(0.4, 1.0, d), rng.standard_normal((d, taps)) * 0.4
        if l["type"] == "hgrn2":
            H, D, E = m["heads"], m["dim"], m["vdim"]
            w.update({q + "q": mat(H * D, d), q + "f": mat(H * D, d), q + "f.b": rng.uniform(-1, 3, H * D), q + "lower": rng.uniform(0, 0.9, H * D), q + "v": mat(H * E, d),
                      q + "norm": rng.uniform(0.6, 1.4, E), q + "o": mat(d, H * E)})
        elif l["type"] == "mlstm":
            H, D, E = m["heads"], m["dim"], m["vdim"]
            w.update({q + "q": mat(H * D, d), q + "k": mat(H * D, d), q + "v": mat(H * E, d), q + "g": mat(H * E, d), q + "o": mat(d, H * E),
                      q + "norm": rng.uniform(0.6, 1.4, H * E), q + "i": mat(H, d), q + "i.b": rng.uniform(-2, 1, H), q + "f": mat(H, d), q + "f.b": rng.uniform(1, 5, H)})
        else:
            a, r = m["left"], m["right"]
            H, G, D, E = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "mix.left."
            w.update({q + "q": mat(H * D, d), q + "k": mat(G * D, d), q + "v": mat(G * E, d), q + "q.b": rng.standard_normal(H * D) * 0.3, q + "k.b": rng.standard_normal(G * D) * 0.3,
                      q + "v.b": rng.standard_normal(G * E) * 0.3, q + "q.norm": rng.uniform(0.6, 1.5, H * D), q + "k.norm": rng.uniform(0.6, 1.5, G * D),
                      q + "sink": rng.uniform(-1.0, 3.0, H), q + "g": mat(H * E, d, 1.5), q + "o": mat(d, H * E, 1.5)})
            h, g, v, n = r["heads"], r["groups"], r["vdim"], r["state"]
            q, inner, channels = p + "mix.right.", h * v, h * v + 2 * g * n
            w.update({q + "in": mat(inner + channels + h, d), q + "conv": rng.standard_normal((channels, r["conv"])) * 0.5, q + "conv.b": rng.standard_normal(channels) * 0.2,
                      q + "dt_bias": rng.uniform(-4, 0, h), q + "A_log": rng.uniform(-1, 1.5, h), q + "D": rng.standard_normal(h), q + "norm": rng.uniform(0.6, 1.4, inner),
                      q + "o": mat(d, inner)})
        if l["mlp"] is not None:
            F, E = l["mlp"]["expert"]["ff"], l["mlp"]["router"]["experts"]
            q = p + "mlp."
            w[p + "norm2"], w[p + "canon2"] = rng.uniform(0.4, 1.0, d), rng.standard_normal((d, taps)) * 0.4
            w[q + "router"], w[q + "correction"] = mat(E, d, 1.5), rng.uniform(-0.3, 0.3, E)
            for e in range(E):
                w.update({q + "e%d.gate" % e: mat(F, d, 1.5), q + "e%d.up" % e: mat(F, d), q + "e%d.down" % e: mat(d, F, 1.5)})
    return rounded(w)


def margin(scores, correction, r):
    """How far the choice of every row is from another one."""
    E, groups, keep, top = r["experts"], r["groups"]["count"], r["groups"]["keep"], r["top"]
    choice = scores + correction
    worth = np.sort(np.sort(choice.reshape(-1, groups, E // groups), axis=-1)[..., -2:].sum(axis=-1), axis=-1)[:, ::-1]
    out = worth[:, keep - 1] - worth[:, keep] if keep < groups else np.full(len(scores), np.inf)
    chosen = to.choose_experts(scores, correction, groups, keep, E // groups * keep)
    ranked = np.take_along_axis(choice, chosen, axis=1)
    return np.minimum(out, ranked[:, top - 1] - ranked[:, top]) if top < E // groups * keep else out


def steady_weights(cfg, seed, least=0.03, codes=8):
    """The same with routers that read nothing but a few coordinates of the token itself, which no sublayer touches, chosen so that no choice is
    close: bfloat16 rounding then changes no expert.  mLSTM layers get smaller input gates."""
    w = random_weights(cfg, seed)
    rng = np.random.default_rng(seed + 1000)
    c = rng.choice(cfg["width"], codes, replace=False)
    routed = [i for i, l in enumerate(cfg["layers"]) if l["mlp"] is not None]
    w["pos"][:, c] = 0.0
    for k in w:
        if k.endswith(("norm1", "norm2")):
            w[k][c] = 0.0
        if k.endswith(("canon1", "canon2")):
            w[k][c] = 0.0
    for k in w:  # input gates that leave the normaliser's floor in place: where n . q alone divides, it now and then is next to nothing
        if k.endswith(".i.b"):
            w[k] -= 2.5
    for i in routed:
        r = w["l%d.mlp.router" % i]
        kept = r[:, c] * np.sqrt(cfg["width"] / codes)
        r[:] = 0.0
        r[:, c] = kept
    w = rounded(w)
    for t in range(cfg["vocab"]):
        best = None
        for _ in range(200):
            code = bf16_to_f32(bf16_bits(rng.uniform(-1.2, 1.2, codes)))
            m = min([np.inf] + [margin(to.sigmoid(code[None].astype(np.float64) @ w["l%d.mlp.router" % i][:, c].T), w["l%d.mlp.correction" % i],
                                       cfg["layers"][i]["mlp"]["router"])[0] for i in routed])
            if best is None or m > best[0]:
                best = (m, code)
            if m > least:
                break
        w["embed"][t, c] = best[1]
    return w
