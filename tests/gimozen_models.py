"""Small random Gimozen models for the tests: configurations, weights, model folders."""
import numpy as np

from tests.nigenex_models import logit_error, write_folder  # noqa: F401  (shared by the tests of both designs)
from turbospark_b200.plain import bf16_bits, bf16_to_f32

YARN = {"factor": 3.0, "original": 400, "fast": 8.0, "slow": 1.0}


def latent(heads, dim, rot_dim, vdim, kv_rank, ff, scale=None, base=5000.0, scaling=YARN, kv_from=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = scaling
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": 1.4 / (dim + rot_dim) ** 0.5 if scale is None else scale,
         "rot": rot}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def attention(heads, kv_heads, dim, vdim, ff, scale=None, temp=(0.4, 37)):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.2 / dim ** 0.5 if scale is None else scale}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, eps=1e-5, alpha=1.7, embed=2.5):
    return {"architecture": "Gimozen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "postln_alpha": alpha, "embedding": {"scale": embed},
            "layers": layers}


# name -> configuration.  Sizes that divide nothing evenly, sizes that happen to be equal or one, layers that differ.
CONFIGS = {
    "odd": config(200, 333, [latent(5, 24, 12, 20, 72, 136), attention(6, 3, 40, 24, 136), latent(7, 18, 12, 33, 72, None, kv_from=0),
                             attention(6, 2, 20, 28, None, temp=None)], eps=1e-3),
    # no scaling of the rotation, no feed-forward, borrowing twice from a latent that is not the last one
    "borrow": config(96, 130, [attention(4, 4, 32, 32, 72, scale=0.12), latent(4, 32, 8, 32, 48, 72, scale=0.15, scaling=None),
                               latent(3, 16, 4, 16, 40, None, base=300.0), latent(6, 20, 8, 12, 48, 72, scale=0.2, scaling=None, kv_from=1),
                               latent(2, 64, 8, 64, 48, 9, scale=0.1, scaling=None, kv_from=1)], alpha=2.0, embed=1.0),
    # a head of 192 columns in expanded form, a value of 128
    "wide_heads": config(160, 97, [latent(3, 100, 60, 72, 130, 64), attention(12, 1, 64, 64, 100), latent(2, 130, 60, 128, 130, 40, kv_from=0)], eps=1e-6),
    # heads that no expanded kernel takes, a latent above 256, key and value sizes above 128
    "large": config(128, 64, [latent(2, 160, 48, 150, 300, 48), attention(4, 2, 130, 200, 32), attention(2, 1, 72, 96, 8)], embed=0.7),
    # many heads over one latent row: more than a query tile holds
    "many_heads": config(128, 75, [latent(40, 8, 6, 8, 30, 64), attention(24, 1, 16, 16, 64, temp=(1.0, 1))]),
    # constants that are one
    "ones": config(96, 60, [attention(2, 2, 16, 16, 32, scale=0.15, temp=(1.0, 1)), latent(2, 16, 4, 16, 24, None, scale=0.15)], alpha=1.0, embed=1.0),
    "single": config(64, 40, [latent(1, 16, 2, 16, 8, 16, scale=0.2), attention(1, 1, 16, 8, 1, scale=0.2)], embed=1.0),
}


def random_weights(cfg, seed):
    """name -> float32 array whose values are bfloat16 numbers."""
    rng = np.random.default_rng(seed)
    d, V = cfg["width"], cfg["vocab"]

    def mat(rows, cols, gain=1.0):
        return rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    w = {"embed": rng.standard_normal((V, d)) * 0.8, "head": mat(V, d, 2.0), "final.norm": rng.uniform(-0.4, 0.4, d)}
    for i, l in enumerate(cfg["layers"]):
        p, m = "l%d." % i, l["mixer"]
        H, D, E = m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"] = rng.uniform(-0.4, 0.4, d)
        if l["type"] == "latent_attention":
            R, K = m["rot_dim"], m["kv_rank"]
            w[p + "mix.q"] = mat(H * (D + R), d)
            if "kv_from" not in m:
                w[p + "mix.dkv"], w[p + "mix.dkv.norm"] = mat(K + R, d, 1.3), rng.uniform(0.6, 1.5, K)
            w[p + "mix.uk"], w[p + "mix.uv"] = mat(H * D, K), mat(H * E, K)
            w[p + "mix.sink"] = rng.uniform(-1.0, 3.0, H)
            w[p + "mix.g"] = mat(H * E, d, 1.5)
        else:
            G = m["kv_heads"]
            w[p + "mix.q"], w[p + "mix.k"], w[p + "mix.v"] = mat(H * D, d), mat(G * D, d), mat(G * E, d)
            w[p + "mix.q.norm"], w[p + "mix.k.norm"] = rng.uniform(0.6, 1.5, D), rng.uniform(0.6, 1.5, D)
        w[p + "mix.o"] = mat(d, H * E, 1.5)
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            w[p + "norm2"] = rng.uniform(-0.4, 0.4, d)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(F, d, 1.5), mat(F, d), mat(d, F, 1.5)
    return {k: bf16_to_f32(bf16_bits(v)).reshape(np.shape(v)) for k, v in w.items()}
