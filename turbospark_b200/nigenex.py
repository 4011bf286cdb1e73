"""The Nigenex design as a plain-weight decoder: its config.json keys and its tensor names.

Parallel layers with one scalar-gain norm, a token shift before the mixer, and sliding-window attention whose values are
its keys, with capped scores, a logarithmic distance bias and one output gate per head; dense gelu feed-forwards (or none);
capped logits.  Every size and constant comes from config.json.
"""
from . import plain
from .plain import need as _need

ARCHITECTURE = "Nigenex"


def parse_config(config, max_context, compute=plain.BF16):
    """config.json's content -> (PlainConfig, [PlainLayer])."""
    layers = []
    for i, entry in enumerate(_need(config, "layers", "the model")):
        where = "layer %d" % i
        kind = _need(entry, "type", where)
        if kind != "attention":
            raise ValueError("config: %s: unknown mixer type '%s'" % (where, kind))
        m = _need(entry, "mixer", where)
        dim, vdim = int(_need(m, "dim", where)), int(_need(m, "vdim", where))
        if vdim != dim:
            raise ValueError("config: %s: the values are the keys, so vdim (%d) must equal dim (%d)" % (where, vdim, dim))
        window = int(_need(_need(m, "mask", where), "size", where))
        if window < 1:
            raise ValueError("config: %s: a window holds at least the token itself" % where)
        mlp = _need(entry, "mlp", where)
        ff = 0
        if mlp is not None:
            if _need(mlp, "kind", where) != "dense":
                raise ValueError("config: %s: unknown feed-forward kind '%s'" % (where, mlp["kind"]))
            ff = int(_need(mlp, "ff", where))
        layers.append(plain.PlainLayer(n_q_heads=int(_need(m, "heads", where)), n_kv_heads=int(_need(m, "kv_heads", where)), head_dim=dim,
                                       window=window, score_scale=float(_need(m, "scale", where)), score_cap=float(_need(m, "softcap", where)),
                                       log_bias=1, head_gate=1, token_shift=1, ffn=ff, act=plain.GELU_TANH))
    cfg = plain.PlainConfig(n_layers=len(layers), d_model=int(_need(config, "width", "the model")), vocab=int(_need(config, "vocab", "the model")),
                            max_context=max_context, compute=compute, norm_eps=float(_need(_need(config, "norm", "the model"), "eps", "norm")),
                            logit_cap=float(_need(config, "logit_softcap", "the model")))
    return cfg, layers


def load_tensors(model, get):
    """Upload every tensor; get(name) returns the array (uint16 = bfloat16 bits)."""
    model.set(plain.P_EMBED, get("embed"))
    model.set(plain.P_HEAD, get("head"))
    model.set(plain.P_FINAL_NORM, get("final.norm"))
    for i, layer in enumerate(model.layers):
        p = "l%d." % i
        names = [(plain.P_NORM, "norm1"), (plain.P_SHIFT, "shift"), (plain.P_Q, "mix.q"), (plain.P_K, "mix.k"), (plain.P_HEAD_GATE, "mix.g"),
                 (plain.P_R1, "mix.r1"), (plain.P_R2, "mix.r2"), (plain.P_O, "mix.o")]
        if layer.ffn:
            names += [(plain.P_FF_GATE, "mlp.gate"), (plain.P_FF_UP, "mlp.up"), (plain.P_FF_DOWN, "mlp.down")]
        for which, name in names:
            model.set(which, get(p + name), layer=i)


def build(ctx, config, get, max_context, compute):
    return plain.build(ctx, *parse_config(config, max_context, compute), load_tensors, get)
