"""The Tarivik design as a plain-weight decoder: its config.json keys and its tensor names.

Output-norm layers (grouped norms of the sublayers' outputs) whose sublayers read the stream through short convolutions, learned
positions, and routed feed-forwards with sigmoid scores and limited expert groups (or none).  Three mixers in any order: HGRN2 and mLSTM
recurrences, and, side by side, chunked attention (projection norms, linear distance bias, sinks, output gates) with a Mamba-2
recurrence.  Every size and constant comes from config.json.
"""
import numpy as np

from . import plain
from .plain import need

ARCHITECTURE = "Tarivik"


def _hgrn2(m, where):
    return dict(recurrence=plain.REC_FORGET, rec_heads=int(need(m, "heads", where)), rec_dim=int(need(m, "dim", where)), rec_vdim=int(need(m, "vdim", where)))


def _mlstm(m, where):
    return dict(recurrence=plain.REC_MLSTM, rec_heads=int(need(m, "heads", where)), rec_dim=int(need(m, "dim", where)), rec_vdim=int(need(m, "vdim", where)),
                rec_cap=float(need(m, "gate_cap", where)))


def _parallel(m, where):
    a, r = need(m, "left", where), need(m, "right", where)
    chunk = int(need(need(a, "mask", where), "size", where))
    if chunk < 1:
        raise ValueError("config: %s: a chunk holds at least the token itself" % where)
    return dict(n_q_heads=int(need(a, "heads", where)), n_kv_heads=int(need(a, "kv_heads", where)), head_dim=int(need(a, "dim", where)),
                value_dim=int(need(a, "vdim", where)), score_scale=float(need(a, "scale", where)), chunk=chunk, qk_norm=plain.NORM_PROJECTION, qkv_bias=1,
                linear_bias=1, sink=1, value_gate=1, attn_scale=float(need(m, "left_scale", where)), rec_scale=float(need(m, "right_scale", where)),
                recurrence=plain.REC_SSD, rec_heads=int(need(r, "heads", where)), rec_dim=int(need(r, "state", where)), rec_vdim=int(need(r, "vdim", where)),
                rec_groups=int(need(r, "groups", where)), rec_taps=int(need(r, "conv", where)), rec_norm_groups=int(need(r, "norm_groups", where)))


MIXERS = {"hgrn2": _hgrn2, "mlstm": _mlstm, "parallel": _parallel}


def parse_config(config, max_context, compute=plain.BF16):
    """config.json's content -> (PlainConfig, [PlainLayer]).  A context ends where the learned positions end."""
    layers = []
    for i, entry in enumerate(need(config, "layers", "the model")):
        where = "layer %d" % i
        kind = need(entry, "type", where)
        if kind not in MIXERS:
            raise ValueError("config: %s: unknown mixer type '%s'" % (where, kind))
        fields = MIXERS[kind](need(entry, "mixer", where), where)
        mlp = need(entry, "mlp", where)
        if mlp is not None:
            if need(mlp, "kind", where) != "moe":
                raise ValueError("config: %s: unknown feed-forward kind '%s'" % (where, mlp["kind"]))
            r = need(mlp, "router", where)
            groups = need(r, "groups", where)
            fields.update(ffn=int(need(need(mlp, "expert", where), "ff", where)), experts=int(need(r, "experts", where)), expert_top=int(need(r, "top", where)),
                          expert_groups=int(need(groups, "count", where)), expert_keep=int(need(groups, "keep", where)))
        layers.append(plain.PlainLayer(act=plain.SILU, **fields))
    norm, positions = need(config, "norm", "the model"), int(need(config, "max_positions", "the model"))
    cfg = plain.PlainConfig(n_layers=len(layers), d_model=int(need(config, "width", "the model")), vocab=int(need(config, "vocab", "the model")),
                            max_context=min(max_context, positions), compute=compute, norm_eps=float(need(norm, "eps", "norm")), output_norm=1,
                            norm_groups=int(need(norm, "groups", "norm")), conv_taps=int(need(need(config, "canon", "the model"), "taps", "canon")),
                            positions=positions)
    return cfg, layers


_MIXER_TENSORS = {
    plain.REC_FORGET: [(plain.P_REC_Q, "q"), (plain.P_REC_F, "f"), (plain.P_REC_F_BIAS, "f.b"), (plain.P_REC_LOWER, "lower"), (plain.P_REC_V, "v"),
                       (plain.P_REC_NORM, "norm"), (plain.P_REC_O, "o")],
    plain.REC_MLSTM: [(plain.P_REC_Q, "q"), (plain.P_REC_K, "k"), (plain.P_REC_V, "v"), (plain.P_REC_GATE, "g"), (plain.P_REC_I, "i"),
                      (plain.P_REC_I_BIAS, "i.b"), (plain.P_REC_F, "f"), (plain.P_REC_F_BIAS, "f.b"), (plain.P_REC_NORM, "norm"), (plain.P_REC_O, "o")],
    plain.REC_SSD: [(plain.P_Q, "left.q"), (plain.P_Q_BIAS, "left.q.b"), (plain.P_K, "left.k"), (plain.P_K_BIAS, "left.k.b"), (plain.P_V, "left.v"),
                    (plain.P_V_BIAS, "left.v.b"), (plain.P_Q_NORM, "left.q.norm"), (plain.P_K_NORM, "left.k.norm"), (plain.P_SINK, "left.sink"),
                    (plain.P_VALUE_GATE, "left.g"), (plain.P_O, "left.o"), (plain.P_REC_IN, "right.in"), (plain.P_REC_CONV, "right.conv"),
                    (plain.P_REC_CONV_BIAS, "right.conv.b"), (plain.P_REC_DT_BIAS, "right.dt_bias"), (plain.P_REC_A_LOG, "right.A_log"),
                    (plain.P_REC_D, "right.D"), (plain.P_REC_NORM, "right.norm"), (plain.P_REC_O, "right.o")],
}


def load_tensors(model, get):
    """Upload every tensor; get(name) returns the array (uint16 = bfloat16 bits)."""
    for which, name in ((plain.P_EMBED, "embed"), (plain.P_POSITIONS, "pos"), (plain.P_HEAD, "head"), (plain.P_FINAL_NORM, "final.norm")):
        model.set(which, get(name))
    taps = model.cfg.conv_taps > 0
    for i, layer in enumerate(model.layers):
        p = "l%d." % i
        names = [(plain.P_NORM, "norm1")] + ([(plain.P_CONV1, "canon1")] if taps else [])
        names += [(which, "mix." + name) for which, name in _MIXER_TENSORS[layer.recurrence]]
        if layer.ffn:
            names += [(plain.P_NORM2, "norm2"), (plain.P_ROUTER, "mlp.router"), (plain.P_CORRECTION, "mlp.correction")]
            names += [(plain.P_CONV2, "canon2")] if taps else []
            for which, name in ((plain.P_FF_GATE, "gate"), (plain.P_FF_UP, "up"), (plain.P_FF_DOWN, "down")):
                model.set(which, np.concatenate([get("%smlp.e%d.%s" % (p, e, name)) for e in range(layer.experts)]), layer=i)
        for which, name in names:
            model.set(which, get(p + name), layer=i)


def build(ctx, config, get, max_context, compute):
    return plain.build(ctx, *parse_config(config, max_context, compute), load_tensors, get)
