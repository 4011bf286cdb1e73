"""ctypes binding of libtsb.so (include/tsb.h)."""
import ctypes as C
import os

import numpy as np

_HERE = os.path.dirname(os.path.abspath(__file__))
Q4_K, Q6_K, MXFP4, Q5_K, Q8_0 = 0, 1, 2, 3, 4

_lib = None
_path = None


def use_library(path):
    """Load this build of the library instead of the in-tree one (before the first call of lib())."""
    global _path
    assert _lib is None or path == _path, "the library is already loaded"
    _path = path


class TsbError(RuntimeError):
    def __init__(self, code, message):
        super().__init__("tsb status %d: %s" % (code, message))
        self.code = code


def lib_path():
    # TSB_LIB points at another build of the same library (kernel experiments); the default is the in-tree one
    return _path or os.environ.get("TSB_LIB") or os.path.join(_HERE, "libtsb.so")


class RowDesc(C.Structure):
    _fields_ = [("seq", C.c_int32), ("base", C.c_int32), ("slot", C.c_int32), ("position", C.c_int32),
                ("mask", C.c_uint64 * 2)]


class Shaping(C.Structure):
    _fields_ = [("temperature", C.c_double), ("top_k", C.c_uint32), ("_pad", C.c_uint32), ("top_p", C.c_double),
                ("repetition_penalty", C.c_double), ("presence_penalty", C.c_double),
                ("frequency_penalty", C.c_double), ("min_p", C.c_double), ("seed", C.c_uint64)]


def shaping(temperature=1.0, top_k=0, top_p=0.0, repetition_penalty=1.0, presence_penalty=0.0,
            frequency_penalty=0.0, min_p=0.0, seed=0):
    return Shaping(temperature, top_k, 0, top_p, repetition_penalty, presence_penalty, frequency_penalty, min_p, seed)


class AcceptOut(C.Structure):
    _fields_ = [("accepted", C.c_int32), ("draws", C.c_int32), ("tokens", C.c_int32 * 16), ("status", C.c_int32),
                ("_pad", C.c_int32), ("margin_accept", C.c_double), ("margin_draw", C.c_double)]


def row_descs(entries):
    """entries: iterable of (seq, base, slot, position, mask_int) -> ctypes array of RowDesc."""
    entries = list(entries)
    arr = (RowDesc * len(entries))()
    for i, (seq, base, slot, position, mask) in enumerate(entries):
        arr[i].seq, arr[i].base, arr[i].slot, arr[i].position = seq, base, slot, position
        arr[i].mask[0] = mask & 0xFFFFFFFFFFFFFFFF
        arr[i].mask[1] = (mask >> 64) & 0xFFFFFFFFFFFFFFFF
    return arr


def lib():
    """Loads libtsb.so; raises if it has not been built (there is no fallback path)."""
    global _lib
    if _lib is None:
        path = lib_path()
        if not os.path.exists(path):
            raise ImportError("libtsb.so is missing: build it with `python -m turbospark_b200.build` "
                              "(no CPU fallback exists)")
        L = C.CDLL(path)
        L.tsb_last_error.restype = C.c_char_p
        L.tsb_last_error.argtypes = [C.c_void_p]
        L.tsb_row_bytes.restype = C.c_int64
        L.tsb_row_bytes.argtypes = [C.c_int32, C.c_int64]
        L.tsb_launch_count.restype = C.c_uint64
        L.tsb_launch_count.argtypes = [C.c_void_p]
        L.tsb_uniform_u64.restype = C.c_uint64
        L.tsb_uniform_u64.argtypes = [C.c_int32, C.c_uint64, C.c_uint64]
        for name in ("tsb_attn_scratch_bytes", "tsb_accept_scratch_bytes", "tsb_accept_history_scratch_bytes", "tsb_gemm_workspace_bytes", "tsb_plain_gemm_workspace_bytes",
                     "tsb_window_attention_scratch_bytes", "tsb_recurrence_scratch_bytes"):
            if hasattr(L, name):
                getattr(L, name).restype = C.c_size_t
        if hasattr(L, "tsb_kv_cursor"):
            L.tsb_kv_cursor.restype = C.c_int64
            L.tsb_kv_cursor.argtypes = [C.c_void_p, C.c_int32]
        _lib = L
    return _lib


def _vp(x):
    if x is None:
        return None
    if isinstance(x, DeviceBuffer):
        return C.c_void_p(x.ptr)
    if isinstance(x, np.ndarray):
        return x.ctypes.data_as(C.c_void_p)
    if isinstance(x, int):
        return C.c_void_p(x)
    return x


class DeviceBuffer:
    """Device memory owned through tsb_alloc / tsb_free."""

    def __init__(self, ctx, nbytes):
        self.ctx = ctx
        self.nbytes = int(nbytes)
        p = C.c_void_p()
        ctx.check(lib().tsb_alloc(ctx.h, C.c_size_t(self.nbytes), C.byref(p)))
        self.ptr = p.value

    def upload(self, arr, stream=None):
        arr = np.ascontiguousarray(arr)
        assert arr.nbytes <= self.nbytes
        self.ctx.check(lib().tsb_memcpy_h2d(self.ctx.h, stream, C.c_void_p(self.ptr), _vp(arr), C.c_size_t(arr.nbytes)))
        self.ctx.sync(stream)
        return self

    def download(self, dtype, count, stream=None, offset=0):
        out = np.empty(count, dtype=dtype)
        self.ctx.check(lib().tsb_memcpy_d2h(self.ctx.h, stream, _vp(out), C.c_void_p(self.ptr + offset),
                                            C.c_size_t(out.nbytes)))
        self.ctx.sync(stream)
        return out

    def free(self):
        if self.ptr:
            lib().tsb_free(self.ctx.h, C.c_void_p(self.ptr))
            self.ptr = 0

    def __del__(self):
        try:
            self.free()
        except Exception:
            pass


class Ctx:
    def __init__(self, device=0):
        h = C.c_void_p()
        rc = lib().tsb_ctx_create(C.c_int32(device), C.byref(h))
        if rc:
            raise TsbError(rc, "tsb_ctx_create failed (no CUDA device, or not an sm_100 GPU)")
        self.h = h

    def check(self, rc):
        if rc:
            raise TsbError(rc, lib().tsb_last_error(self.h).decode())

    def sync(self, stream=None):
        self.check(lib().tsb_stream_sync(self.h, stream))

    def alloc(self, nbytes):
        return DeviceBuffer(self, nbytes)

    def to_device(self, arr):
        if isinstance(arr, C.Array):
            arr = np.frombuffer(bytes(arr), dtype=np.uint8)
        arr = np.ascontiguousarray(arr)
        return DeviceBuffer(self, max(arr.nbytes, 16)).upload(arr)

    def upload_weights(self, arr):
        arr = np.ascontiguousarray(arr, dtype=np.uint8)
        p = C.c_void_p()
        self.check(lib().tsb_weights_upload(self.h, _vp(arr), C.c_size_t(arr.nbytes), C.byref(p)))
        b = DeviceBuffer.__new__(DeviceBuffer)
        b.ctx, b.nbytes, b.ptr = self, arr.nbytes, p.value
        return b

    @property
    def launches(self):
        return int(lib().tsb_launch_count(self.h))

    def set_wait_limit_us(self, microseconds):
        """Bound of every wait inside a kernel; when it runs out the kernel reports an error and returns."""
        self.check(lib().tsb_ctx_set_wait_limit_us(self.h, C.c_uint32(microseconds)))

    def debug_wait_nobody(self, out_u32, stream=None):
        self.check(lib().tsb_debug_wait_nobody(self.h, stream, _vp(out_u32)))

    # ---- operators
    def gemm_quant(self, qtype, w, rows, cols, x, y, tokens, y_f32=False, w_off=0, stream=None):
        self.check(lib().tsb_gemm_quant(self.h, stream, C.c_int32(qtype), _vp(w), C.c_uint64(w_off), C.c_int64(rows),
                                        C.c_int64(cols), _vp(x), _vp(y), C.c_int32(tokens), C.c_int32(int(y_f32))))

    def gemm_workspace_bytes(self, qtype, rows, cols, tokens):
        return int(lib().tsb_gemm_workspace_bytes(C.c_int32(qtype), C.c_int64(rows), C.c_int64(cols), C.c_int32(tokens)))

    def gemm_prepare(self, qtype, rows, cols, x, tokens, workspace, stream=None):
        self.check(lib().tsb_gemm_prepare(self.h, stream, C.c_int32(qtype), C.c_int64(rows), C.c_int64(cols), _vp(x), C.c_int32(tokens),
                                          _vp(workspace), C.c_size_t(workspace.nbytes)))

    def gemm_quant_prepared(self, qtype, w, rows, cols, x, workspace, y, tokens, y_f32=False, w_off=0, stream=None):
        self.check(lib().tsb_gemm_quant_prepared(self.h, stream, C.c_int32(qtype), _vp(w), C.c_uint64(w_off), C.c_int64(rows),
                                                 C.c_int64(cols), _vp(x), _vp(workspace), _vp(y), C.c_int32(tokens), C.c_int32(int(y_f32))))

    def dequant_rows(self, qtype, w, cols, row_ids, n_rows, out, w_off=0, stream=None):
        self.check(lib().tsb_dequant_rows(self.h, stream, C.c_int32(qtype), _vp(w), C.c_uint64(w_off), C.c_int64(cols),
                                          _vp(row_ids), C.c_int32(n_rows), _vp(out)))

    def embed_rows(self, qtype, w, vocab_rows, cols, token_ids, n, out, out_scale=1.0, w_off=0, stream=None):
        self.check(lib().tsb_embed_rows(self.h, stream, C.c_int32(qtype), _vp(w), C.c_uint64(w_off),
                                        C.c_int64(vocab_rows), C.c_int64(cols), _vp(token_ids), C.c_int32(n), _vp(out),
                                        C.c_float(out_scale)))

    def rmsnorm_rows(self, x, residual, w_bf16, out, rows, d, eps, stream=None):
        self.check(lib().tsb_rmsnorm_rows(self.h, stream, _vp(x), _vp(residual), _vp(w_bf16), _vp(out), C.c_int32(rows),
                                          C.c_int32(d), C.c_float(eps)))

    def rope_rows(self, x, rows, heads, head_dim, rotated_pairs, row_stride, positions, theta, stream=None):
        self.check(lib().tsb_rope_neox_rows_positions(self.h, stream, _vp(x), C.c_int32(rows), C.c_int32(heads),
                                                      C.c_int32(head_dim), C.c_int32(rotated_pairs),
                                                      C.c_int64(row_stride), _vp(positions), C.c_float(theta)))

    def silu_mul(self, gate, up, out, rows, n, in_stride, out_stride, stream=None):
        self.check(lib().tsb_silu_mul(self.h, stream, _vp(gate), _vp(up), _vp(out), C.c_int32(rows), C.c_int32(n),
                                      C.c_int64(in_stride), C.c_int64(out_stride)))

    def attn_scratch_bytes(self, rows, n_q_heads, head_dim):
        return int(lib().tsb_attn_scratch_bytes(C.c_int32(rows), C.c_int32(n_q_heads), C.c_int32(head_dim)))

    def rope_store_kv(self, kv, layer, qkv, rows_dev, rows, n_q_heads, theta, stream=None):
        self.check(lib().tsb_rope_store_kv(self.h, stream, kv.h, C.c_int32(layer), _vp(qkv), _vp(rows_dev),
                                           C.c_int32(rows), C.c_int32(n_q_heads), C.c_float(theta)))

    def attn_decode_rows(self, kv, layer, q, q_stride, out, rows_dev, rows, rows_per_seq, n_q_heads, scale, max_len,
                         scratch, stream=None):
        self.check(lib().tsb_attn_decode_rows(self.h, stream, kv.h, C.c_int32(layer), _vp(q), C.c_int64(q_stride),
                                              _vp(out), _vp(rows_dev), C.c_int32(rows), C.c_int32(rows_per_seq),
                                              C.c_int32(n_q_heads), C.c_float(scale), C.c_int32(max_len), _vp(scratch),
                                              C.c_size_t(scratch.nbytes)))

    def attn_decode_rows_static(self, kv, layer, q, q_stride, out, rows_dev, rows, rows_per_seq, n_q_heads, scale, max_len,
                                stream=None):
        """tsb_attn_decode_rows with the library's built-in scratch area (no buffer argument, no allocation)."""
        self.check(lib().tsb_attn_decode_rows_static(self.h, stream, kv.h, C.c_int32(layer), _vp(q), C.c_int64(q_stride),
                                                     _vp(out), _vp(rows_dev), C.c_int32(rows), C.c_int32(rows_per_seq),
                                                     C.c_int32(n_q_heads), C.c_float(scale), C.c_int32(max_len)))

    def accept_scratch_bytes(self, batch, k, vocab):
        return int(lib().tsb_accept_scratch_bytes(C.c_int32(batch), C.c_int32(k), C.c_int32(vocab)))

    def accept(self, target_logits, draft_logits, proposals, uniforms, batch, k, vocab, shaping_cfg, out, scratch,
               stream=None):
        self.check(lib().tsb_accept(self.h, stream, _vp(target_logits), _vp(draft_logits), _vp(proposals), _vp(uniforms),
                                    C.c_int32(batch), C.c_int32(k), C.c_int32(vocab), C.byref(shaping_cfg), _vp(out),
                                    _vp(scratch), C.c_size_t(scratch.nbytes)))

    def sample(self, logits, uniforms, batch, vocab, shaping_cfg, tokens, margins, scratch, stream=None):
        self.check(lib().tsb_sample(self.h, stream, _vp(logits), _vp(uniforms), C.c_int32(batch), C.c_int32(vocab),
                                    C.byref(shaping_cfg), _vp(tokens), _vp(margins), _vp(scratch),
                                    C.c_size_t(scratch.nbytes)))

    def accept_history_scratch_bytes(self, batch, k, vocab):
        return int(lib().tsb_accept_history_scratch_bytes(C.c_int32(batch), C.c_int32(k), C.c_int32(vocab)))

    def accept_history(self, target_logits, draft_logits, proposals, uniforms, batch, k, vocab, shaping_cfg, history, hist_stride,
                       hist_len, generated, out, scratch, stream=None):
        """tsb_accept with the history penalties: history [batch, hist_stride] i32, hist_len / generated [batch] i32 (device)."""
        self.check(lib().tsb_accept_history(self.h, stream, _vp(target_logits), _vp(draft_logits), _vp(proposals), _vp(uniforms),
                                            C.c_int32(batch), C.c_int32(k), C.c_int32(vocab), C.byref(shaping_cfg), _vp(history),
                                            C.c_int32(hist_stride), _vp(hist_len), _vp(generated), _vp(out), _vp(scratch),
                                            C.c_size_t(scratch.nbytes)))

    def sample_history(self, logits, uniforms, batch, vocab, shaping_cfg, history, hist_stride, hist_len, generated, tokens, margins,
                       scratch, stream=None):
        self.check(lib().tsb_sample_history(self.h, stream, _vp(logits), _vp(uniforms), C.c_int32(batch), C.c_int32(vocab),
                                            C.byref(shaping_cfg), _vp(history), C.c_int32(hist_stride), _vp(hist_len), _vp(generated),
                                            _vp(tokens), _vp(margins), _vp(scratch), C.c_size_t(scratch.nbytes)))

    def moe_route(self, router_logits, tokens, n_experts, k, ids_out, weights_out, scale=None, stream=None):
        self.check(lib().tsb_moe_route(self.h, stream, _vp(router_logits), C.c_int32(tokens), C.c_int32(n_experts), C.c_int32(k),
                                       _vp(scale) if scale is not None else None, _vp(ids_out), _vp(weights_out)))

    def router_logits(self, q_u8, scale_bf16, bias_bf16, x, tokens, n_experts, d_model, logits_out, stream=None):
        self.check(lib().tsb_router_logits(self.h, stream, _vp(q_u8), _vp(scale_bf16), _vp(bias_bf16), _vp(x), C.c_int32(tokens),
                                           C.c_int32(n_experts), C.c_int32(d_model), _vp(logits_out)))

    def moe_ffn(self, qtype, gate_up, down, n_experts, d_model, ffn, x, residual, ids, weights, tokens, k, y, stream=None):
        self.check(lib().tsb_moe_ffn(self.h, stream, C.c_int32(qtype), _vp(gate_up), C.c_uint64(0), _vp(down), C.c_uint64(0),
                                     C.c_int32(n_experts), C.c_int32(d_model), C.c_int32(ffn), _vp(x), _vp(residual), _vp(ids),
                                     _vp(weights), C.c_int32(tokens), C.c_int32(k), _vp(y)))

    # ---- plain-weight operators (type: 0 bfloat16, 1 f32)
    def zeroed(self, nbytes):
        return self.to_device(np.zeros(nbytes, dtype=np.uint8))

    def plain_gemm_workspace(self):
        return self.zeroed(int(lib().tsb_plain_gemm_workspace_bytes(self.h)))

    def window_attention_scratch(self):
        return self.zeroed(int(lib().tsb_window_attention_scratch_bytes(self.h)))

    def plain_gemm(self, type_, w, rows, cols, x, x_rows, tokens, y, y_stride, n_valid, workspace, cap=0.0, add=False, stream=None):
        self.check(lib().tsb_plain_gemm(self.h, stream, C.c_int32(type_), _vp(w), C.c_int64(rows), C.c_int64(cols), _vp(x), C.c_int32(x_rows),
                                        C.c_int32(tokens), _vp(y), C.c_int64(y_stride), C.c_int32(n_valid), C.c_float(cap), C.c_int32(int(add)),
                                        _vp(workspace)))

    def plain_gemm_pairs(self, type_, w, rows, cols, x, x_rows, tokens, a, a_stride, n_pairs, act, workspace, stream=None):
        self.check(lib().tsb_plain_gemm_pairs(self.h, stream, C.c_int32(type_), _vp(w), C.c_int64(rows), C.c_int64(cols), _vp(x), C.c_int32(x_rows),
                                              C.c_int32(tokens), _vp(a), C.c_int64(a_stride), C.c_int32(n_pairs), C.c_int32(act), _vp(workspace)))

    def norm_shift_rows(self, type_, x, d, gain, eps, mu, rows_dev, rows, state, n_streams, ring, mix_out, h_out, out_stride, stream=None):
        self.check(lib().tsb_norm_shift_rows(self.h, stream, C.c_int32(type_), _vp(x), C.c_int32(d), _vp(gain), C.c_float(eps), _vp(mu), _vp(rows_dev),
                                             C.c_int32(rows), _vp(state), C.c_int32(n_streams), C.c_int32(ring), _vp(mix_out), _vp(h_out),
                                             C.c_int64(out_stride)))

    def window_attention(self, kv, layer, q, q_stride, out, out_stride, rows_dev, group_rows, n_q_heads, scale, cap, r1, r2, gate, window, max_len,
                         scratch, stream=None):
        gr = (C.c_int32 * len(group_rows))(*group_rows)
        self.check(lib().tsb_window_attention(self.h, stream, kv.h, C.c_int32(layer), _vp(q), C.c_int64(q_stride), _vp(out), C.c_int64(out_stride),
                                              _vp(rows_dev), gr, C.c_int32(len(group_rows)), C.c_int32(n_q_heads), C.c_float(scale), C.c_float(cap),
                                              _vp(r1), _vp(r2), _vp(gate), C.c_int32(window), C.c_int32(max_len), _vp(scratch)))

    def plain_attention(self, kv, layer, q, q_stride, out, out_stride, rows_dev, group_rows, n_q_heads, scale, max_len, scratch, stream=None, cap=0.0,
                        window=0, r1=None, r2=None, head_gate=None, sink=None, value_gate=None, value_gate_stride=0, slopes=None, chunk=0, out_scale=0.0,
                        keep=0, blocks=False, turn=None, turn_half=0):
        gr = (C.c_int32 * len(group_rows))(*group_rows)
        x = AttentionExtras(cap, window, _vp(r1), _vp(r2), _vp(head_gate), _vp(sink), _vp(value_gate), value_gate_stride,
                            _vp(slopes), chunk, out_scale, keep, int(blocks), _vp(turn), turn_half)
        self.check(lib().tsb_plain_attention(self.h, stream, kv.h, C.c_int32(layer), _vp(q), C.c_int64(q_stride), _vp(out), C.c_int64(out_stride),
                                             _vp(rows_dev), gr, C.c_int32(len(group_rows)), C.c_int32(n_q_heads), C.c_float(scale), C.byref(x),
                                             C.c_int32(max_len), _vp(scratch)))

    def latent_attention(self, kv, layer, q, q_stride, out, out_stride, rows_dev, group_rows, n_heads, value_dim, scale, sink, max_len, scratch,
                         stream=None):
        gr = (C.c_int32 * len(group_rows))(*group_rows)
        self.check(lib().tsb_latent_attention(self.h, stream, kv.h, C.c_int32(layer), _vp(q), C.c_int64(q_stride), _vp(out), C.c_int64(out_stride),
                                              _vp(rows_dev), gr, C.c_int32(len(group_rows)), C.c_int32(n_heads), C.c_int32(value_dim), C.c_float(scale),
                                              _vp(sink), C.c_int32(max_len), _vp(scratch)))

    def plain_gemm_heads(self, type_, w, heads, head_rows, cols, x, x_stride, x_step, x_rows, tokens, y, y_stride, y_step, n_valid, workspace, gate=None,
                         gate_stride=0, gate_step=0, stream=None):
        self.check(lib().tsb_plain_gemm_heads(self.h, stream, C.c_int32(type_), _vp(w), C.c_int32(heads), C.c_int32(head_rows), C.c_int64(cols), _vp(x),
                                              C.c_int64(x_stride), C.c_int32(x_step), C.c_int32(x_rows), C.c_int32(tokens), _vp(y), C.c_int64(y_stride),
                                              C.c_int32(y_step), C.c_int32(n_valid), _vp(gate), C.c_int64(gate_stride), C.c_int32(gate_step),
                                              _vp(workspace)))

    def post_norm_rows(self, type_, x, d, weight, eps, rows, out, out_stride, stream=None):
        self.check(lib().tsb_post_norm_rows(self.h, stream, C.c_int32(type_), _vp(x), C.c_int32(d), _vp(weight), C.c_float(eps), C.c_int32(rows), _vp(out),
                                            C.c_int64(out_stride)))

    def pre_norm_rows(self, type_, x, d, weight, eps, rows, out, out_stride, stream=None):
        self.check(lib().tsb_pre_norm_rows(self.h, stream, C.c_int32(type_), _vp(x), C.c_int32(d), _vp(weight), C.c_float(eps), C.c_int32(rows), _vp(out),
                                           C.c_int64(out_stride)))

    def turned_norm_rows(self, kv, layer, raw, raw_stride, n_q, n_k, width, q_weight, k_weight, eps, rows_dev, rows, q, q_stride, rot=None, rot_half=0, n_v=0, v_width=0,
                         turn=None, turn_half=0, projection=False, stream=None):
        n = TurnedNorms(int(projection), n_q, n_k, n_v, width, v_width, rot_half, turn_half, _vp(raw), _vp(q_weight), _vp(k_weight), _vp(rot), _vp(turn), raw_stride, q_stride,
                        _vp(q), eps)
        self.check(lib().tsb_turned_norm_rows(self.h, stream, kv.h, C.c_int32(layer), C.byref(n), _vp(rows_dev), C.c_int32(rows)))

    def block_mean_rows(self, kv, layer, rows_dev, rows, stream=None):
        self.check(lib().tsb_block_mean_rows(self.h, stream, kv.h, C.c_int32(layer), _vp(rows_dev), C.c_int32(rows)))

    def gated_scan_rows(self, type_, gate, gate_stride, out_gate, out_gate_stride, width, state, n_streams, ring, rows_dev, rows, rows_per_seq, out, out_stride, chunked=False, sums=None,
                        stream=None):
        self.check(lib().tsb_gated_scan_rows(self.h, stream, C.c_int32(type_), _vp(gate), C.c_int64(gate_stride), _vp(out_gate), C.c_int64(out_gate_stride), C.c_int32(width),
                                             _vp(state), C.c_int32(n_streams), C.c_int32(ring), _vp(rows_dev), C.c_int32(rows), C.c_int32(rows_per_seq), C.c_int32(int(chunked)),
                                             _vp(sums), _vp(out), C.c_int64(out_stride)))

    def plain_gemm_act(self, type_, w, rows, cols, x, x_rows, tokens, y, y_stride, n_valid, act, workspace, stream=None):
        self.check(lib().tsb_plain_gemm_act(self.h, stream, C.c_int32(type_), _vp(w), C.c_int64(rows), C.c_int64(cols), _vp(x), C.c_int32(x_rows), C.c_int32(tokens), _vp(y),
                                            C.c_int64(y_stride), C.c_int32(n_valid), C.c_int32(act), _vp(workspace)))

    def plain_gemm_add(self, type_, w, rows, cols, x, x_rows, tokens, y, y_stride, n_valid, alpha, beta, workspace, stream=None):
        self.check(lib().tsb_plain_gemm_add(self.h, stream, C.c_int32(type_), _vp(w), C.c_int64(rows), C.c_int64(cols), _vp(x), C.c_int32(x_rows), C.c_int32(tokens), _vp(y),
                                            C.c_int64(y_stride), C.c_int32(n_valid), C.c_float(alpha), C.c_float(beta), _vp(workspace)))

    def head_norm_rows(self, kv, layer, raw, raw_stride, n_q, n_k, width, q_weight, k_weight, eps, rows_dev, rows, q, q_stride, temp_coef=0.0, temp_every=0,
                       stream=None):
        self.check(lib().tsb_head_norm_rows(self.h, stream, kv.h, C.c_int32(layer), _vp(raw), C.c_int64(raw_stride), C.c_int32(n_q), C.c_int32(n_k),
                                            C.c_int32(width), _vp(q_weight), _vp(k_weight), C.c_float(eps), C.c_float(temp_coef), C.c_int32(temp_every),
                                            _vp(rows_dev), C.c_int32(rows), _vp(q), C.c_int64(q_stride)))

    def output_norm_rows(self, type_, x_in, y, d, weight, groups, eps, taps_w, taps, state, n_streams, ring, rows_dev, rows, rows_per_seq, x_out, out, out_stride,
                         before=None, stream=None):
        self.check(lib().tsb_output_norm_rows(self.h, stream, C.c_int32(type_), _vp(x_in), _vp(y), C.c_int32(d), _vp(weight), C.c_int32(groups), C.c_float(eps),
                                              _vp(taps_w), C.c_int32(taps), _vp(state), _vp(before), C.c_int32(n_streams), C.c_int32(ring), _vp(rows_dev),
                                              C.c_int32(rows), C.c_int32(rows_per_seq), _vp(x_out), _vp(out), C.c_int64(out_stride)))

    def projection_norm_rows(self, kv, layer, raw, raw_stride, n_q, n_k, width, q_weight, k_weight, eps, rows_dev, rows, q, q_stride, stream=None):
        self.check(lib().tsb_projection_norm_rows(self.h, stream, kv.h, C.c_int32(layer), _vp(raw), C.c_int64(raw_stride), C.c_int32(n_q), C.c_int32(n_k),
                                                  C.c_int32(width), _vp(q_weight), _vp(k_weight), C.c_float(eps), _vp(rows_dev), C.c_int32(rows), _vp(q),
                                                  C.c_int64(q_stride)))

    def short_conv_rows(self, type_, x, x_stride, channels, taps_w, taps, bias, state, n_streams, ring, rows_dev, rows, rows_per_seq, out, out_stride, before=None,
                        stream=None):
        self.check(lib().tsb_short_conv_rows(self.h, stream, C.c_int32(type_), _vp(x), C.c_int64(x_stride), C.c_int32(channels), _vp(taps_w), C.c_int32(taps),
                                             _vp(bias), _vp(state), _vp(before), C.c_int32(n_streams), C.c_int32(ring), _vp(rows_dev), C.c_int32(rows),
                                             C.c_int32(rows_per_seq), _vp(out), C.c_int64(out_stride)))

    def recurrence_scratch(self, kind, heads, dim, vdim, rows, rows_per_seq):
        return self.zeroed(int(lib().tsb_recurrence_scratch_bytes(C.c_int32(kind), C.c_int32(heads), C.c_int32(dim), C.c_int32(vdim), C.c_int32(rows),
                                                                  C.c_int32(rows_per_seq))))

    def recurrence_rows(self, type_, rec, rows_dev, rows, rows_per_seq, chunked=False, stream=None):
        self.check(lib().tsb_recurrence_rows(self.h, stream, C.c_int32(type_), C.byref(rec), _vp(rows_dev), C.c_int32(rows), C.c_int32(rows_per_seq),
                                             C.c_int32(int(chunked))))

    def gated_norm_rows(self, type_, o, o_stride, width, groups, weight, weight_n, eps, rows, out, out_stride, scale=1.0, pre_gate=None, post_gate=None, gate_stride=0,
                        stream=None):
        self.check(lib().tsb_gated_norm_rows(self.h, stream, C.c_int32(type_), _vp(o), C.c_int64(o_stride), C.c_int32(width), C.c_int32(groups), _vp(weight),
                                             C.c_int32(weight_n), C.c_float(eps), C.c_float(scale), _vp(pre_gate), _vp(post_gate), C.c_int64(gate_stride),
                                             C.c_int32(rows), _vp(out), C.c_int64(out_stride)))

    def route_experts(self, logits, correction, experts, top, groups, keep, rows, chunk_slots, lists, stream=None):
        self.check(lib().tsb_route_experts(self.h, stream, _vp(logits), _vp(correction), C.c_int32(experts), C.c_int32(top), C.c_int32(groups), C.c_int32(keep),
                                           C.c_int32(rows), C.c_int32(chunk_slots), C.byref(lists.c)))

    def plain_gemm_experts(self, type_, w, experts, w_rows, cols, x, x_stride, x_rows, by_token, lists, slots, chunk_slots, tensor, pairs, y, y_stride, n_valid,
                           stream=None):
        self.check(lib().tsb_plain_gemm_experts(self.h, stream, C.c_int32(type_), _vp(w), C.c_int32(experts), C.c_int64(w_rows), C.c_int64(cols), _vp(x),
                                                C.c_int64(x_stride), C.c_int32(x_rows), C.c_int32(int(by_token)), C.byref(lists.c), C.c_int32(slots),
                                                C.c_int32(chunk_slots), C.c_int32(int(tensor)), C.c_int32(int(pairs)), _vp(y), C.c_int64(y_stride),
                                                C.c_int32(n_valid)))

    def residual_add(self, x, y, n, stream=None):
        self.check(lib().tsb_residual_add(self.h, stream, _vp(x), _vp(y), C.c_int64(n)))

    def close(self):
        if getattr(self, "h", None):
            lib().tsb_ctx_destroy(self.h)
            self.h = None

    def __del__(self):
        pass  # explicit close only: buffers may outlive the Python object order at interpreter exit


class KvCache:
    def __init__(self, ctx, layers, kv_heads, head_dim, page_tokens, num_pages, max_seqs, max_pages_per_seq):
        self.ctx = ctx
        self.layers, self.kv_heads, self.head_dim = layers, kv_heads, head_dim
        h = C.c_void_p()
        ctx.check(lib().tsb_kv_create(ctx.h, C.c_int32(layers), C.c_int32(kv_heads), C.c_int32(head_dim),
                                      C.c_int32(page_tokens), C.c_int32(num_pages), C.c_int32(max_seqs),
                                      C.c_int32(max_pages_per_seq), C.byref(h)))
        self.h = h

    def reserve(self, seq, tokens):
        self.ctx.check(lib().tsb_kv_reserve(self.h, C.c_int32(seq), C.c_int64(tokens)))

    def reset(self, seq):
        self.ctx.check(lib().tsb_kv_reset(self.h, C.c_int32(seq)))

    def cursor(self, seq):
        return int(lib().tsb_kv_cursor(self.h, C.c_int32(seq)))

    def set_cursor(self, seq, pos):
        self.ctx.check(lib().tsb_kv_set_cursor(self.h, C.c_int32(seq), C.c_int64(pos)))

    def rewind_by(self, seq, count):
        self.ctx.check(lib().tsb_kv_rewind_by(self.h, C.c_int32(seq), C.c_int64(count)))

    def write_rows(self, seq, layer, pos0, k, v, stream=None):
        k = np.ascontiguousarray(k, dtype=np.uint16)
        v = np.ascontiguousarray(v, dtype=np.uint16)
        n = k.size // (self.kv_heads * self.head_dim)
        self.ctx.check(lib().tsb_kv_write_rows(self.h, stream, C.c_int32(seq), C.c_int32(layer), C.c_int64(pos0),
                                               C.c_int32(n), _vp(k), _vp(v)))

    def read_rows(self, seq, layer, pos0, n, stream=None):
        k = np.empty((n, self.kv_heads * self.head_dim), dtype=np.uint16)
        v = np.empty_like(k)
        self.ctx.check(lib().tsb_kv_read_rows(self.h, stream, C.c_int32(seq), C.c_int32(layer), C.c_int64(pos0),
                                              C.c_int32(n), _vp(k), _vp(v)))
        return k, v

    def fill_random(self, seq, tokens, seed, stream=None):
        self.ctx.check(lib().tsb_kv_fill_random(self.h, stream, C.c_int32(seq), C.c_int64(tokens), C.c_uint64(seed)))

    def commit_path(self, seq, base, path, stream=None):
        p = np.ascontiguousarray(path, dtype=np.uint32)
        self.ctx.check(lib().tsb_kv_commit_path(self.ctx.h, stream, self.h, C.c_int32(seq), C.c_int64(base), _vp(p),
                                                C.c_int32(p.size)))

    def close(self):
        if getattr(self, "h", None):
            lib().tsb_kv_destroy(self.h)
            self.h = None


class Recurrence(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("kind", "heads", "dim", "vdim", "heads_per_key")] + [("cap", C.c_float), ("q_scale", C.c_float)] + \
               [(n, C.c_void_p) for n in ("q", "k", "v")] + [(n, C.c_int64) for n in ("q_stride", "k_stride", "v_stride")] + \
               [("gate", C.c_void_p), ("gate_stride", C.c_int64)] + [(n, C.c_void_p) for n in ("lower", "a_log", "skip", "out")] + \
               [("out_stride", C.c_int64)] + [(n, C.c_void_p) for n in ("state", "norm", "top")] + [("ring", C.c_int32), ("n_streams", C.c_int32), ("scratch", C.c_void_p)]


class _ExpertLists(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("ids", "weight", "slot_of", "token_of", "first", "chunks", "n_chunks")]


class ExpertLists:
    """Device buffers of a routed pass."""

    def __init__(self, ctx, rows, top, experts):
        n = rows * top * 4
        self.buffers = {"ids": ctx.zeroed(n), "weight": ctx.zeroed(n), "slot_of": ctx.zeroed(n), "token_of": ctx.zeroed(n), "first": ctx.zeroed(4 * (experts + 1)),
                        "chunks": ctx.zeroed(12 * (experts + rows * top // 8 + 1)), "n_chunks": ctx.zeroed(4)}
        self.c = _ExpertLists(**{k: _vp(b) for k, b in self.buffers.items()})

    def free(self):
        for b in self.buffers.values():
            b.free()


class AttentionExtras(C.Structure):
    _fields_ = [("cap", C.c_float), ("window", C.c_int32)] + [(n, C.c_void_p) for n in ("r1", "r2", "head_gate", "sink", "value_gate")] + \
               [("value_gate_stride", C.c_int64), ("slopes", C.c_void_p), ("chunk", C.c_int32), ("out_scale", C.c_float), ("keep", C.c_int32), ("blocks", C.c_int32),
                ("turn", C.c_void_p), ("turn_half", C.c_int32)]


class TurnedNorms(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("projection", "n_q", "n_k", "n_v", "width", "v_width", "rot_half", "turn_half")] + \
               [(n, C.c_void_p) for n in ("raw", "q_weight", "k_weight", "rot", "turn")] + [("raw_stride", C.c_int64), ("q_stride", C.c_int64), ("q", C.c_void_p), ("eps", C.c_float)]


class PlainCache(KvCache):
    """A plain cache: rows of kv_heads * [key, value] (value_dim 0: the values are the keys), bfloat16 bit patterns (type 0) or f32
    values (type 1).  pool > 0: beside them a row for every block of so many positions."""

    def __init__(self, ctx, type_, layers, kv_heads, key_dim, value_dim, page_tokens, num_pages, max_seqs, max_pages_per_seq, pool=0):
        self.ctx, self.type = ctx, type_
        self.layers, self.kv_heads, self.head_dim = layers, kv_heads, key_dim + value_dim
        h = C.c_void_p()
        ctx.check(lib().tsb_kv_create_blocks(ctx.h, C.c_int32(type_), C.c_int32(layers), C.c_int32(kv_heads), C.c_int32(key_dim), C.c_int32(value_dim),
                                            C.c_int32(pool), C.c_int32(page_tokens), C.c_int32(num_pages), C.c_int32(max_seqs), C.c_int32(max_pages_per_seq), C.byref(h)))
        self.h = h

    def write_rows(self, seq, layer, pos0, k, stream=None):
        k = np.ascontiguousarray(k, dtype=np.float32 if self.type else np.uint16)
        self.ctx.check(lib().tsb_kv_write_rows(self.h, stream, C.c_int32(seq), C.c_int32(layer), C.c_int64(pos0),
                                               C.c_int32(k.size // (self.kv_heads * self.head_dim)), _vp(k), None))

    def read_rows(self, seq, layer, pos0, n, stream=None):
        k = np.empty((n, self.kv_heads * self.head_dim), dtype=np.float32 if self.type else np.uint16)
        self.ctx.check(lib().tsb_kv_read_rows(self.h, stream, C.c_int32(seq), C.c_int32(layer), C.c_int64(pos0), C.c_int32(n), _vp(k), None))
        return k

    def read_blocks(self, seq, layer, block0, n, stream=None):
        k = np.empty((n, self.kv_heads * self.head_dim), dtype=np.float32 if self.type else np.uint16)
        self.ctx.check(lib().tsb_kv_read_blocks(self.h, stream, C.c_int32(seq), C.c_int32(layer), C.c_int64(block0), C.c_int32(n), _vp(k)))
        return k


class KeyCache(PlainCache):
    """A key-only cache: the head size must be one that the attention kernels work on."""

    def __init__(self, ctx, type_, layers, kv_heads, head_dim, page_tokens, num_pages, max_seqs, max_pages_per_seq):
        self.ctx, self.type = ctx, type_
        self.layers, self.kv_heads, self.head_dim = layers, kv_heads, head_dim
        h = C.c_void_p()
        ctx.check(lib().tsb_kv_create_keys(ctx.h, C.c_int32(type_), C.c_int32(layers), C.c_int32(kv_heads), C.c_int32(head_dim), C.c_int32(page_tokens),
                                           C.c_int32(num_pages), C.c_int32(max_seqs), C.c_int32(max_pages_per_seq), C.byref(h)))
        self.h = h
