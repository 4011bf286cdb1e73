"""The Gimozen design as a plain-weight decoder: its config.json keys and its tensor names.

Sequential layers normed after each sum, the stream scaled before it.  Two mixers in any order: latent attention (a low-rank cached
latent and one shared rotated key part, YaRN-scaled rotary positions, a sink per head, an output gate per column; a layer may borrow
an earlier layer's latent), and grouped-query attention without positions whose queries and keys are normed per head and whose
queries grow with the logarithm of the position.  Dense silu feed-forwards (or none).  Every size and constant comes from
config.json.
"""
from . import plain
from .plain import need

ARCHITECTURE = "Gimozen"


def _rotation(m, where):
    rot = need(m, "rot", where)
    dims, rot_dim = int(need(rot, "dims", where)), int(need(m, "rot_dim", where))
    if dims != rot_dim:
        raise ValueError("config: %s: the rotated part is rotated as a whole, so rot.dims (%d) must equal rot_dim (%d)" % (where, dims, rot_dim))
    out = dict(rot_dim=rot_dim, rot_base=float(need(rot, "base", where)))
    scaling = rot.get("scaling")
    if scaling is not None:
        out.update({"rot_" + k: float(need(scaling, k, where)) for k in ("factor", "original", "fast", "slow")})
        if out["rot_factor"] <= 0 or out["rot_original"] <= 0 or out["rot_fast"] <= 0 or out["rot_slow"] <= 0:
            raise ValueError("config: %s: the constants of a rotation's scaling are positive" % where)
    return out


def _latent(m, i, where):
    fields = dict(n_q_heads=int(need(m, "heads", where)), n_kv_heads=1, head_dim=int(need(m, "dim", where)), value_dim=int(need(m, "vdim", where)),
                  kv_rank=int(need(m, "kv_rank", where)), score_scale=float(need(m, "scale", where)), sink=1, value_gate=1, **_rotation(m, where))
    source = m.get("kv_from")
    if source is not None:
        if not 0 <= int(source) < i:
            raise ValueError("config: %s: kv_from (%s) must name an earlier layer" % (where, source))
        fields["kv_source"] = int(source) + 1
    return fields


def _attention(m, where):
    fields = dict(n_q_heads=int(need(m, "heads", where)), n_kv_heads=int(need(m, "kv_heads", where)), head_dim=int(need(m, "dim", where)),
                  value_dim=int(need(m, "vdim", where)), score_scale=float(need(m, "scale", where)), qk_norm=1)
    temp = m.get("q_temp")
    if temp is not None:
        every = need(temp, "every", where)
        if int(every) != every or every < 1:
            raise ValueError("config: %s: q_temp.every is a positive whole number" % where)
        fields.update(q_temp_every=int(every), q_temp_coef=float(need(temp, "coef", where)))
    return fields


def parse_config(config, max_context, compute=plain.BF16):
    """config.json's content -> (PlainConfig, [PlainLayer])."""
    layers = []
    for i, entry in enumerate(need(config, "layers", "the model")):
        where = "layer %d" % i
        kind, m = need(entry, "type", where), need(entry, "mixer", where)
        if kind == "latent_attention":
            fields = _latent(m, i, where)
        elif kind == "attention":
            fields = _attention(m, where)
        else:
            raise ValueError("config: %s: unknown mixer type '%s'" % (where, kind))
        mlp = need(entry, "mlp", where)
        if mlp is not None:
            if need(mlp, "kind", where) != "dense":
                raise ValueError("config: %s: unknown feed-forward kind '%s'" % (where, mlp["kind"]))
            fields["ffn"] = int(need(mlp, "ff", where))
        layers.append(plain.PlainLayer(act=plain.SILU, **fields))
    for i, l in enumerate(layers):
        if l.kv_source:
            o = layers[l.kv_source - 1]
            same = ("kv_rank", "rot_dim", "rot_base", "rot_factor", "rot_original", "rot_fast", "rot_slow")
            if o.kv_source or any(getattr(o, k) != getattr(l, k) for k in same):
                raise ValueError("config: layer %d: kv_from names layer %d, which has no latent like its own" % (i, l.kv_source - 1))
    cfg = plain.PlainConfig(n_layers=len(layers), d_model=int(need(config, "width", "the model")), vocab=int(need(config, "vocab", "the model")),
                            max_context=max_context, compute=compute, norm_eps=float(need(need(config, "norm", "the model"), "eps", "norm")),
                            post_norm=1, residual_scale=float(need(config, "postln_alpha", "the model")),
                            embed_scale=float(need(need(config, "embedding", "the model"), "scale", "embedding")))
    return cfg, layers


def load_tensors(model, get):
    """Upload every tensor; get(name) returns the array (uint16 = bfloat16 bits)."""
    model.set(plain.P_EMBED, get("embed"))
    model.set(plain.P_HEAD, get("head"))
    model.set(plain.P_FINAL_NORM, get("final.norm"))
    for i, layer in enumerate(model.layers):
        names = [(plain.P_NORM, "norm1"), (plain.P_Q, "mix.q"), (plain.P_O, "mix.o")]
        if layer.kv_rank:
            names += [(plain.P_UK, "mix.uk"), (plain.P_UV, "mix.uv"), (plain.P_SINK, "mix.sink"), (plain.P_VALUE_GATE, "mix.g")]
            if not layer.kv_source:
                names += [(plain.P_DKV, "mix.dkv"), (plain.P_DKV_NORM, "mix.dkv.norm")]
        else:
            names += [(plain.P_K, "mix.k"), (plain.P_V, "mix.v"), (plain.P_Q_NORM, "mix.q.norm"), (plain.P_K_NORM, "mix.k.norm")]
        if layer.ffn:
            names += [(plain.P_NORM2, "norm2"), (plain.P_FF_GATE, "mlp.gate"), (plain.P_FF_UP, "mlp.up"), (plain.P_FF_DOWN, "mlp.down")]
        for which, name in names:
            model.set(which, get("l%d.%s" % (i, name)), layer=i)


def build(ctx, config, get, max_context, compute):
    return plain.build(ctx, *parse_config(config, max_context, compute), load_tensors, get)
