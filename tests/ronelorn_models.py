"""Small random Ronelorn models for the tests: configurations, weights, model folders."""
import copy

import numpy as np

from tests.nigenex_models import logit_error, write_folder  # noqa: F401  (shared by the tests of the designs)
from turbospark_b200.plain import bf16_bits, bf16_to_f32


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def pooled(heads, kv_heads, dim, vdim, window, pool, mlp, rot, factor=None, base=1000.0, cap=9.0, scale=None):
    """Attention over a window and means of the blocks before it; rot: how many columns of a head turn."""
    r = {"base": base, "dims": rot}
    if factor is not None:
        r["scaling"] = {"factor": factor}
    return {"type": "attention", "mlp": dense(mlp), "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "pool": pool}, "rot": r,
                                                              "scale": 1.6 / dim ** 0.5 if scale is None else scale, "softcap": cap}}


def kept(heads, kv_heads, dim, vdim, window, keep, mlp, rot, base=700.0, scale=None):
    """Attention over a window and the first tokens."""
    return {"type": "attention_2", "mlp": dense(mlp), "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "keep_first": keep},
                                                                "rot": {"base": base, "dims": rot}, "scale": 1.6 / dim ** 0.5 if scale is None else scale}}


def mingru(width, mlp=None):
    return {"type": "mingru", "mlp": dense(mlp), "mixer": {"width": width}}


def again(j, entry):
    return dict(copy.deepcopy(entry), weights_of=j)


def config(width, vocab, layers, mult=0.6, eps=1e-5, embed=1.3):
    return {"architecture": "Ronelorn", "width": width, "vocab": vocab, "embedding": {"scale": embed}, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


_P = pooled(6, 3, 40, 24, 37, 5, 88, rot=20, factor=2.5)
_K = kept(6, 2, 24, 36, 50, 7, 72, rot=24)
_E = pooled(8, 2, 64, 64, 70, 16, 128, rot=64)
# name -> configuration.  Sizes that divide nothing evenly, sizes that happen to be equal or one, layers that use others' tensors.
CONFIGS = {
    "odd": config(200, 333, [_P, mingru(136), _K, again(0, _P), mingru(57, mlp=40), again(2, _K)], eps=1e-3),
    # heads of the tensor kernels, whole vectors everywhere
    "even": config(256, 130, [_E, kept(4, 1, 128, 128, 130, 66, 192, rot=32), mingru(256), again(0, _E)], mult=1.0),
    # heads that no tensor kernel takes; blocks longer than a page; more kept tokens than the window has; tensors of a later layer
    "large": config(96, 64, [again(2, mingru(300)), pooled(2, 1, 160, 130, 90, 70, 48, rot=6, factor=8.0), mingru(300), kept(3, 3, 250, 8, 20, 100, None, rot=10)], mult=0.3),
    # windows and kept tokens that no prompt of the tests leaves; many heads per key head
    "near": config(128, 75, [pooled(12, 1, 20, 28, 1000, 3, 40, rot=4, cap=3.0), kept(16, 2, 32, 32, 600, 800, 24, rot=2), kept(5, 5, 48, 16, 33, 0, None, rot=16)], embed=1.0),
    # constants and sizes that are one
    "ones": config(64, 40, [pooled(1, 1, 8, 2, 1, 1, 8, rot=2, factor=1.0, cap=1.0), kept(1, 1, 8, 1, 1, 1, 1, rot=2), mingru(1, mlp=3), mingru(8)], mult=1.0, embed=4.0),
}


def rounded(w):
    return {k: bf16_to_f32(bf16_bits(v)).reshape(np.shape(v)) for k, v in w.items()}


def random_weights(cfg, seed):
    """name -> float32 array whose values are bfloat16 numbers."""
    rng = np.random.default_rng(seed)
    d, V = cfg["width"], cfg["vocab"]

    def mat(rows, cols, gain=1.0):
        return rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    w = {"embed": rng.standard_normal((V, d)), "head": mat(V, d, 2.0), "final.norm": rng.uniform(-0.4, 0.4, d)}
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        p, m = "l%d." % i, l["mixer"]
        q = p + "mix."
        w[p + "norm1"] = rng.uniform(-0.4, 0.4, d)
        if l["type"] == "mingru":
            E = m["width"]  # gates that keep much of the state
            w.update({q + "z": mat(E, d, 1.5), q + "z.b": rng.uniform(-5, 0, E), q + "x": mat(E, d, 1.5), q + "x.b": rng.standard_normal(E), q + "g": mat(E, d, 1.5),
                      q + "o": mat(d, E, 2.0)})
        else:
            H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            per = (1, 1) if l["type"] == "attention" else (H, G)
            w.update({q + "q": mat(H * D, d), q + "k": mat(G * D, d), q + "v": mat(G * E, d), q + "q.norm": rng.uniform(0.6, 1.5, per[0] * D),
                      q + "k.norm": rng.uniform(0.6, 1.5, per[1] * D), q + "o": mat(d, H * E, 2.0)})
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            w.update({p + "norm2": rng.uniform(-0.4, 0.4, d), p + "mlp.up": mat(F, d), p + "mlp.down": mat(d, F)})
    return rounded(w)
