"""Small random Nigenex models for the tests: configurations, weights, model folders."""
import json
import os

import numpy as np

from turbospark_b200 import safetensors
from turbospark_b200.plain import bf16_bits, bf16_to_f32


def layer(heads, kv_heads, dim, window, ff, scale=None, softcap=8.0):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": window},
                      "scale": 2.0 / dim ** 0.5 if scale is None else scale, "softcap": softcap},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, eps=1e-5, logit_softcap=12.0):
    return {"architecture": "Nigenex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": logit_softcap, "layers": layers}


# name -> configuration.  Sizes that divide nothing evenly, sizes that happen to be equal or one, layers that differ.
CONFIGS = {
    "odd": config(200, 333, [layer(6, 3, 40, 37, 136), layer(6, 3, 40, 37, 136)], eps=1e-3, logit_softcap=4.0),
    "one_kv": config(96, 130, [layer(5, 1, 24, 16, 72), layer(5, 1, 24, 16, 72)]),
    "mha_wide": config(192, 257, [layer(3, 3, 96, 70, 320), layer(3, 3, 96, 1, 320)]),
    "mixed_layers": config(128, 96, [layer(4, 2, 64, 65, None), layer(8, 1, 32, 2, 100), layer(2, 2, 128, 500, 8), layer(12, 4, 20, 129, None)]),
    "large_heads": config(160, 64, [layer(2, 1, 160, 50, 48), layer(1, 1, 250, 90, 1)], eps=1e-6),
    "single": config(64, 40, [layer(1, 1, 16, 9, 16, softcap=0.7)]),
}


def random_weights(cfg, seed):
    """name -> float32 array whose values are bfloat16 numbers."""
    rng = np.random.default_rng(seed)
    d, V = cfg["width"], cfg["vocab"]

    def mat(rows, cols, gain=1.0):
        return rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    w = {"embed": rng.standard_normal((V, d)) * 1.5, "head": mat(V, d, 2.0), "final.norm": np.array(rng.uniform(0.7, 1.4))}
    for i, l in enumerate(cfg["layers"]):
        p, m = "l%d." % i, l["mixer"]
        H, G, D = m["heads"], m["kv_heads"], m["dim"]
        w[p + "norm1"] = np.array(rng.uniform(0.7, 1.4))
        w[p + "shift"] = rng.uniform(0.0, 1.0, d)
        w[p + "mix.q"], w[p + "mix.k"] = mat(H * D, d), mat(G * D, d)
        w[p + "mix.g"] = mat(H, d, 1.5)
        w[p + "mix.r1"], w[p + "mix.r2"] = rng.uniform(0.02, 1.5, H), rng.uniform(0.05, 0.6, H)
        w[p + "mix.o"] = mat(d, H * D, 1.5)
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(F, d, 1.5), mat(F, d), mat(d, F, 1.5)
    return {k: bf16_to_f32(bf16_bits(v)).reshape(np.shape(v)) for k, v in w.items()}


def write_folder(path, cfg, weights):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    safetensors.write(os.path.join(path, "model.safetensors"), {k: bf16_bits(v).reshape(np.shape(v)) for k, v in weights.items()})


def logit_error(got, want):
    """Per row: rms over the vocabulary of the difference (mean taken off), relative to the rms of all wanted logits."""
    d = np.asarray(got, dtype=np.float64) - want
    d = d - d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / np.sqrt((np.asarray(want) ** 2).mean())
