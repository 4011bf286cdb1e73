"""Binding of the plain-weight decoders (tsb_model_create_plain): layers put together from mechanisms, bfloat16 or f32."""
import ctypes as C

import numpy as np

from .capi import lib
from .model import Model

BF16, F32 = 0, 1
GELU_TANH, SILU, RELU2 = 0, 1, 2
SINK_TENSOR, SINK_ZERO = 1, 2
(P_EMBED, P_HEAD, P_FINAL_NORM, P_NORM, P_SHIFT, P_Q, P_K, P_HEAD_GATE, P_R1, P_R2, P_O, P_FF_GATE, P_FF_UP,
 P_FF_DOWN, P_NORM2, P_V, P_Q_NORM, P_K_NORM, P_SINK, P_VALUE_GATE, P_DKV, P_DKV_NORM, P_UK, P_UV, P_POSITIONS, P_CONV1, P_CONV2, P_Q_BIAS,
 P_K_BIAS, P_V_BIAS, P_ROUTER, P_CORRECTION, P_REC_Q, P_REC_K, P_REC_V, P_REC_GATE, P_REC_F, P_REC_F_BIAS, P_REC_LOWER, P_REC_I, P_REC_I_BIAS, P_REC_NORM,
 P_REC_O, P_REC_IN, P_REC_CONV, P_REC_CONV_BIAS, P_REC_DT_BIAS, P_REC_A_LOG, P_REC_D) = range(49)
NORM_HEAD, NORM_PROJECTION = 1, 2
REC_FORGET, REC_MLSTM, REC_SSD, REC_MINGRU = 1, 2, 3, 4


class PlainConfig(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("n_layers", "d_model", "vocab", "max_context", "compute")] + \
               [("norm_eps", C.c_float), ("logit_cap", C.c_float), ("post_norm", C.c_int32), ("residual_scale", C.c_float),
                ("embed_scale", C.c_float)] + [(n, C.c_int32) for n in ("output_norm", "norm_groups", "conv_taps", "positions", "pre_norm")] + \
               [("sublayer_scale", C.c_float)]


class PlainLayer(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("n_q_heads", "n_kv_heads", "head_dim", "window")] + \
               [("score_scale", C.c_float), ("score_cap", C.c_float)] + \
               [(n, C.c_int32) for n in ("log_bias", "head_gate", "token_shift", "ffn", "act", "value_dim", "qk_norm", "q_temp_every")] + \
               [("q_temp_coef", C.c_float)] + \
               [(n, C.c_int32) for n in ("sink", "value_gate", "kv_rank", "rot_dim", "kv_source")] + \
               [(n, C.c_double) for n in ("rot_base", "rot_factor", "rot_original", "rot_fast", "rot_slow")] + \
               [(n, C.c_int32) for n in ("qkv_bias", "linear_bias", "chunk")] + [(n, C.c_float) for n in ("attn_scale", "rec_scale")] + \
               [(n, C.c_int32) for n in ("recurrence", "rec_heads", "rec_dim", "rec_vdim", "rec_groups", "rec_taps", "rec_norm_groups")] + \
               [("rec_cap", C.c_float)] + [(n, C.c_int32) for n in ("experts", "expert_top", "expert_groups", "expert_keep",
                                                                        "keep_first", "pool", "value_rot", "ff_plain", "weights_of")]


def need(d, key, where):
    """The value of a key that a configuration must have."""
    if not isinstance(d, dict) or key not in d:
        raise ValueError("config: %s has no '%s'" % (where, key))
    return d[key]


def bf16_bits(x):
    """float32 -> bfloat16 bit patterns, round to nearest even."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_to_f32(bits):
    return (np.asarray(bits, dtype=np.uint16).astype(np.uint32) << 16).view(np.float32)


class PlainModel(Model):
    def __init__(self, ctx, cfg, layers):
        self.ctx, self.cfg, self.layers = ctx, cfg, list(layers)
        arr = (PlainLayer * len(self.layers))(*self.layers)
        h = C.c_void_p()
        ctx.check(lib().tsb_model_create_plain(ctx.h, C.byref(cfg), arr, C.byref(h)))
        self.h = h

    def set(self, which, array, layer=-1):
        """Upload one tensor: uint16 arrays are bfloat16 bit patterns, anything else is taken as float32."""
        a = np.asarray(array)
        host = BF16 if a.dtype == np.uint16 else F32
        a = np.ascontiguousarray(a, dtype=np.uint16 if host == BF16 else np.float32)
        rows, cols = a.shape if a.ndim == 2 else (1, a.size)
        self.ctx.check(lib().tsb_model_set_plain(self.h, C.c_int32(layer), C.c_int32(which), C.c_int32(host), a.ctypes.data_as(C.c_void_p),
                                                 C.c_int64(rows), C.c_int64(cols)))

    def fill(self, seed=0):
        """Seeded random weights made on the device."""
        self.ctx.check(lib().tsb_model_fill_plain(self.h, C.c_uint64(seed)))


def build(ctx, cfg, layers, load_tensors, get):
    """A model with its tensors: load_tensors(model, get) uploads what get(name) returns."""
    model = PlainModel(ctx, cfg, layers)
    try:
        load_tensors(model, get)
    except Exception:
        model.close()
        raise
    return model
