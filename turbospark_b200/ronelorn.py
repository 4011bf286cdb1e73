"""The Ronelorn design as a plain-weight decoder: its config.json keys and its tensor names.

Pre-norm layers whose sublayers are scaled before they join the stream.  Three mixers in any order: attention over a window and, before it, over
means of blocks of keys and values (norms per head, scaled rotary positions, values that turn with their position, capped scores); attention over
a window and the first tokens (norms of whole projections, rotary positions, a sink of score zero); a minGRU recurrence.  Dense feed-forwards
with squared relu and no gate (or none).  A layer may use another layer's tensors.  Every size and constant comes from config.json.
"""
from . import plain
from .plain import need

ARCHITECTURE = "Ronelorn"


def _rotation(m, where):
    rot = need(m, "rot", where)
    out = dict(rot_dim=int(need(rot, "dims", where)), rot_base=float(need(rot, "base", where)))
    if out["rot_dim"] % 2 or not 0 <= out["rot_dim"] <= int(need(m, "dim", where)):
        raise ValueError("config: %s: rot.dims (%d) is an even part of a head" % (where, out["rot_dim"]))
    scaling = rot.get("scaling")
    if scaling is not None:
        out["rot_factor"] = float(need(scaling, "factor", where))
        if out["rot_factor"] <= 0:
            raise ValueError("config: %s: rot.scaling.factor is positive" % where)
    return out


def _heads(m, where):
    window = int(need(need(m, "mask", where), "size", where))
    if window < 1:
        raise ValueError("config: %s: a window holds at least the token itself" % where)
    return dict(n_q_heads=int(need(m, "heads", where)), n_kv_heads=int(need(m, "kv_heads", where)), head_dim=int(need(m, "dim", where)),
                value_dim=int(need(m, "vdim", where)), score_scale=float(need(m, "scale", where)), window=window, **_rotation(m, where))


def _pooled(m, where):
    pool = int(need(m["mask"], "pool", where)) if "mask" in m else 0
    fields = _heads(m, where)
    if pool < 1:
        raise ValueError("config: %s: a block holds at least one token" % where)
    if fields["value_dim"] % 2:
        raise ValueError("config: %s: values are turned in pairs, so vdim (%d) is even" % (where, fields["value_dim"]))
    return dict(qk_norm=plain.NORM_HEAD, value_rot=1, pool=pool, score_cap=float(need(m, "softcap", where)), **fields)


def _kept(m, where):
    fields = _heads(m, where)
    keep = int(need(m["mask"], "keep_first", where))
    if keep < 0:
        raise ValueError("config: %s: keep_first must not be negative" % where)
    return dict(qk_norm=plain.NORM_PROJECTION, sink=plain.SINK_ZERO, keep_first=keep, **fields)


def _mingru(m, where):
    return dict(recurrence=plain.REC_MINGRU, rec_heads=1, rec_dim=1, rec_vdim=int(need(m, "width", where)))


MIXERS = {"attention": _pooled, "attention_2": _kept, "mingru": _mingru}


def _owner(entries, i):
    """The layer whose tensors layer i uses."""
    seen = {i}
    while entries[i].get("weights_of") is not None:
        j = int(entries[i]["weights_of"])
        if not 0 <= j < len(entries) or j in seen:
            raise ValueError("config: layer %d: weights_of (%d) names no layer with tensors" % (i, j))
        seen.add(j)
        i = j
    return i


def parse_config(config, max_context, compute=plain.BF16):
    """config.json's content -> (PlainConfig, [PlainLayer])."""
    entries, layers = need(config, "layers", "the model"), []
    for i, entry in enumerate(entries):
        where = "layer %d" % i
        kind = need(entry, "type", where)
        if kind not in MIXERS:
            raise ValueError("config: %s: unknown mixer type '%s'" % (where, kind))
        fields = MIXERS[kind](need(entry, "mixer", where), where)
        mlp = need(entry, "mlp", where)
        if mlp is not None:
            if need(mlp, "kind", where) != "dense":
                raise ValueError("config: %s: unknown feed-forward kind '%s'" % (where, mlp["kind"]))
            fields.update(ffn=int(need(mlp, "ff", where)), ff_plain=1)
        owner = _owner(entries, i)
        if owner != i:
            fields["weights_of"] = owner + 1
        layers.append(plain.PlainLayer(act=plain.RELU2, **fields))
    for i, l in enumerate(layers):
        o = layers[l.weights_of - 1] if l.weights_of else l
        differ = [n for n, _ in plain.PlainLayer._fields_ if n != "weights_of" and getattr(o, n) != getattr(l, n)]
        if differ:
            raise ValueError("config: layer %d differs from layer %d, whose tensors it uses (%s)" % (i, l.weights_of - 1, ", ".join(differ)))
    mult = float(need(config, "residual_mult", "the model"))
    if mult == 0:
        raise ValueError("config: residual_mult must not be zero")
    cfg = plain.PlainConfig(n_layers=len(layers), d_model=int(need(config, "width", "the model")), vocab=int(need(config, "vocab", "the model")),
                            max_context=max_context, compute=compute, norm_eps=float(need(need(config, "norm", "the model"), "eps", "norm")), pre_norm=1,
                            sublayer_scale=mult, embed_scale=float(need(need(config, "embedding", "the model"), "scale", "embedding")))
    return cfg, layers


_ATTENTION = [(plain.P_Q, "q"), (plain.P_K, "k"), (plain.P_V, "v"), (plain.P_Q_NORM, "q.norm"), (plain.P_K_NORM, "k.norm"), (plain.P_O, "o")]
_MINGRU = [(plain.P_REC_F, "z"), (plain.P_REC_F_BIAS, "z.b"), (plain.P_REC_I, "x"), (plain.P_REC_I_BIAS, "x.b"), (plain.P_REC_GATE, "g"), (plain.P_REC_O, "o")]


def load_tensors(model, get):
    """Upload every tensor; get(name) returns the array (uint16 = bfloat16 bits)."""
    for which, name in ((plain.P_EMBED, "embed"), (plain.P_HEAD, "head"), (plain.P_FINAL_NORM, "final.norm")):
        model.set(which, get(name))
    for i, layer in enumerate(model.layers):
        if layer.weights_of:
            continue
        names = [(plain.P_NORM, "norm1")] + [(which, "mix." + name) for which, name in (_MINGRU if layer.recurrence else _ATTENTION)]
        if layer.ffn:
            names += [(plain.P_NORM2, "norm2"), (plain.P_FF_UP, "mlp.up"), (plain.P_FF_DOWN, "mlp.down")]
        for which, name in names:
            model.set(which, get("l%d.%s" % (i, name)), layer=i)


def build(ctx, config, get, max_context, compute):
    return plain.build(ctx, *parse_config(config, max_context, compute), load_tensors, get)
