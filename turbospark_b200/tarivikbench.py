"""Prefill and decode throughput of Tarivik-shaped models beside Gimozen-shaped ones of equal size, and the time of each kernel against
its roofline beside the like kernel (python bench.py --design tarivik).  Method as in plainbench.
"""
import ctypes as C

import numpy as np

from . import capi, latentbench, plainbench
from .model import Session
from .plain import BF16, NORM_PROJECTION, REC_FORGET, REC_MLSTM, REC_SSD, SILU, PlainConfig, PlainLayer, PlainModel
from .plainbench import L2_BYTES, Peaks, decode, on_stream, plain_matmul, random_bf16, time_graph, visible

# Equal to latentbench's shapes in width, attention heads, layers, vocabulary and the feed-forward width that a token meets.
# attention: query heads, key heads, head size; ssd: heads, columns, state, groups; forget and mlstm: heads, dim, columns;
# experts: how many, how many taken, width, groups, groups kept
SHAPES = {"8b": dict(d=4096, layers=32, vocab=128256, norm_groups=8, attention=(32, 8, 128), ssd=(64, 64, 128, 8), forget=(32, 128, 128), mlstm=(32, 64, 128),
                     experts=(32, 8, 1792, 8, 4)),
          "2b": dict(d=2048, layers=16, vocab=128256, norm_groups=4, attention=(32, 8, 64), ssd=(32, 64, 128, 4), forget=(16, 128, 128), mlstm=(16, 64, 128),
                     experts=(32, 8, 1024, 8, 4))}
TAPS, CHUNK, RING = 4, 8192, 8


def _f32(ctx, n, seed, lo=-1.0, hi=1.0):
    return ctx.to_device(np.random.default_rng(seed).uniform(lo, hi, size=n).astype(np.float32))


def _rows(ctx, context, rows, streams):
    return ctx.to_device(capi.row_descs([(s, context, j, context + j, 0) for s in range(streams) for j in range(rows)]))


def attention(ctx, peaks, name, nq, nkv, hd, context, rows, streams, iters):
    """Chunked attention with slopes, sinks and output gates."""
    kv, layers = latentbench._cache(ctx, nkv, hd, hd, context, rows, streams)
    n = streams * rows
    q, out, rd = random_bf16(ctx, n * nq * hd, 3, amp=3.5), ctx.alloc(n * nq * hd * 2), _rows(ctx, context, rows, streams)
    sink, slopes, gate = ctx.zeroed(nq * 4), ctx.to_device((2.0 ** (-8.0 * (np.arange(nq) + 1) / nq)).astype(np.float32)), random_bf16(ctx, n * nq * hd, 4)
    scratch = ctx.window_attention_scratch()
    ms = time_graph(lambda i, s: ctx.plain_attention(kv, i % layers, q, nq * hd, out, nq * hd, rd, [rows] * streams, nq, hd ** -0.5, context + rows, scratch, sink=sink,
                                                     slopes=slopes, value_gate=gate, value_gate_stride=nq * hd, chunk=CHUNK, stream=s), iters)
    seen, distinct = visible(context, rows, 0)
    kv.close()
    for b in (q, out, rd, sink, slopes, gate, scratch):
        b.free()
    return dict(peaks.entry(name, ms, streams * distinct * nkv * 2 * hd * 2 + n * nq * 3 * hd * 2, 4.0 * hd * nq * seen * streams), context=context, rows=rows, streams=streams)


def recurrence(ctx, peaks, kind, heads, dim, vdim, rows, streams, iters, groups=0):
    """Per-stream states are read and written once; vectors and gates of every row are read, outputs written."""
    keys = groups or heads
    n, kd, inner = streams * rows, keys * dim, heads * vdim
    gates = {REC_FORGET: heads * dim, REC_MLSTM: 2 * heads, REC_SSD: heads}[kind]
    state_bytes = heads * dim * vdim * 4
    copies = max(2, -(-2 * L2_BYTES // (2 * state_bytes * streams))) if rows < 64 else max(2, -(-2 * L2_BYTES // (n * (2 * kd + inner) * 2)))
    copies = min(copies, 64)
    q, k, v = (random_bf16(ctx, copies * n * w, s, amp=1.0) for w, s in ((kd, 1), (kd, 2), (inner, 3)))
    gate = ctx.to_device(np.random.default_rng(4).standard_normal(n * gates).astype(np.float32) + (3.0 if kind != REC_SSD else 0.0))
    lower, a_log, skip = _f32(ctx, heads * dim, 5, 0.0, 0.9), _f32(ctx, heads, 6), _f32(ctx, heads, 7)
    out, state = ctx.alloc(n * inner * 4), [ctx.zeroed(streams * 2 * state_bytes) for _ in range(copies if rows < 64 else 1)]
    copies_ = (vdim + 31) // 32
    norm, top, rd = ctx.zeroed(streams * 2 * heads * copies_ * dim * 4), ctx.zeroed(streams * 2 * heads * copies_ * 8), _rows(ctx, 0 if rows >= 64 else 4096, rows, streams)

    scratch = ctx.recurrence_scratch(kind, heads, dim, vdim, n, rows) if rows >= 64 else ctx.zeroed(16)

    def call(i, s):
        at = i % copies
        r = capi.Recurrence(kind=kind, heads=heads, dim=dim, vdim=vdim, heads_per_key=heads // keys, cap=15.0, q_scale=dim ** -0.5 if kind == REC_MLSTM else 0.0,
                            q=q.ptr + at * n * kd * 2, k=k.ptr + at * n * kd * 2, v=v.ptr + at * n * inner * 2, q_stride=kd, k_stride=kd, v_stride=inner, gate=gate.ptr,
                            gate_stride=gates, lower=lower.ptr, a_log=a_log.ptr, skip=skip.ptr, out=out.ptr, out_stride=inner, state=state[i % len(state)].ptr,
                            norm=norm.ptr, top=top.ptr, ring=2, n_streams=streams, scratch=scratch.ptr)
        ctx.recurrence_rows(BF16, r, rd, n, rows, chunked=rows >= 64, stream=s)
    ms = time_graph(call, iters)
    for b in [q, k, v, gate, lower, a_log, skip, out, norm, top, rd, scratch] + state:
        b.free()
    vectors = (kd if kind == REC_FORGET else 2 * kd) + inner
    nbytes = streams * state_bytes * (2 if rows < 64 else 1) + n * (2 * vectors + 4 * gates + 4 * inner)
    name = {REC_FORGET: "recurrence, decay per channel", REC_MLSTM: "recurrence, mLSTM", REC_SSD: "recurrence, Mamba-2"}[kind]
    return dict(peaks.entry(name, ms, nbytes, 4.0 * n * heads * dim * vdim), rows=rows, streams=streams)


def output_norm(ctx, peaks, name, d, groups, rows, iters):
    copies = max(2, -(-2 * L2_BYTES // (rows * d * 14))) if rows > 256 else 2
    x, y = [_f32(ctx, rows * d, i) for i in range(copies)], [_f32(ctx, rows * d, 9 + i) for i in range(copies)]
    x2, out = [ctx.alloc(rows * d * 4) for _ in range(copies)], [ctx.alloc(rows * d * 2) for _ in range(copies)]
    w, taps, state, before, rd = _f32(ctx, d, 1), _f32(ctx, d * TAPS, 2), ctx.zeroed(RING * d * 4), ctx.zeroed((TAPS - 1) * d * 4), _rows(ctx, 0, rows, 1)
    ms = time_graph(lambda i, s: ctx.output_norm_rows(BF16, x[i % copies], y[i % copies], d, w, groups, 1e-6, taps, TAPS, state, 1, RING, rd, rows, rows,
                                                      x2[i % copies], out[i % copies], d, before=before, stream=s), iters)
    for b in x + y + x2 + out + [w, taps, state, before, rd]:
        b.free()
    return dict(peaks.entry(name, ms, rows * d * 14.0), rows=rows, d=d)


def projection_norms(ctx, peaks, name, nq, nk, hd, rows, iters):
    kv, layers = latentbench._cache(ctx, nk, hd, hd, 0, rows, 1)
    per = (nq + nk) * hd
    copies = max(2, -(-2 * L2_BYTES // (rows * per * 6))) if rows > 256 else 2
    raws, qs = [ctx.zeroed(rows * per * 4) for _ in range(copies)], [ctx.alloc(rows * nq * hd * 2) for _ in range(copies)]
    w, rd = ctx.zeroed(nq * hd * 4), _rows(ctx, 0, rows, 1)
    ms = time_graph(lambda i, s: ctx.projection_norm_rows(kv, i % layers, raws[i % copies], per, nq, nk, hd, w, w, 1e-6, rd, rows, qs[i % copies], nq * hd, stream=s), iters)
    kv.close()
    for b in raws + qs + [w, rd]:
        b.free()
    return dict(peaks.entry(name, ms, rows * per * 6.0), rows=rows)


def short_conv(ctx, peaks, name, channels, rows, iters):
    copies = max(2, -(-2 * L2_BYTES // (rows * channels * 4))) if rows > 256 else 2
    x, out = random_bf16(ctx, copies * rows * channels, 1), ctx.alloc(copies * rows * channels * 2)
    w, bias, state, before, rd = _f32(ctx, channels * TAPS, 2), _f32(ctx, channels, 3), ctx.zeroed(RING * channels * 4), ctx.zeroed(3 * channels * 4), _rows(ctx, 0, rows, 1)

    def call(i, s):
        at = (i % copies) * rows * channels * 2
        ctx.short_conv_rows(BF16, C.c_void_p(x.ptr + at), channels, channels, w, TAPS, bias, state, 1, RING, rd, rows, rows, C.c_void_p(out.ptr + at), channels,
                            before=before, stream=s)
    ms = time_graph(call, iters)
    for b in (x, out, w, bias, state, before, rd):
        b.free()
    return dict(peaks.entry(name, ms, rows * channels * 4.0), rows=rows, channels=channels)


def gated_norm(ctx, peaks, name, width, groups, rows, iters):
    copies = max(2, -(-2 * L2_BYTES // (rows * width * 8))) if rows > 256 else 2
    o, gate, out = [_f32(ctx, rows * width, i) for i in range(copies)], random_bf16(ctx, rows * width, 1), [ctx.alloc(rows * width * 2) for _ in range(copies)]
    w = _f32(ctx, width, 3)
    ms = time_graph(lambda i, s: ctx.gated_norm_rows(BF16, o[i % copies], width, width, groups, w, width, 1e-6, rows, out[i % copies], width, pre_gate=gate,
                                                     gate_stride=width, stream=s), iters)
    for b in o + out + [gate, w]:
        b.free()
    return dict(peaks.entry(name, ms, rows * width * 8.0), rows=rows, width=width)


def experts(ctx, peaks, d, shape, tokens, iters):
    """Choice and lists; the two grouped products over as many slots (an expert's matrices count once if a token meets it)."""
    n, top, ff, groups, keep = shape
    slots, few = tokens * top, 8 if tokens <= 8 else 16
    tensor = tokens > 16 and slots >= 12 * n
    logits, corr, lists = ctx.to_device(np.random.default_rng(1).standard_normal((tokens, n)).astype(np.float32)), _f32(ctx, n, 2, -0.1, 0.1), capi.ExpertLists(ctx, tokens, top, n)
    route = time_graph(lambda i, s: ctx.route_experts(logits, corr, n, top, groups, keep, tokens, few, lists, stream=s), iters)
    ids = np.empty(slots, dtype=np.int32)
    ctx.check(capi.lib().tsb_memcpy_d2h(ctx.h, None, ids.ctypes.data_as(C.c_void_p), C.c_void_p(lists.buffers["ids"].ptr), C.c_size_t(ids.nbytes)))
    ctx.sync()
    met = len(np.unique(ids))
    ff_pad = (ff + 63) // 64 * 64
    copies = max(2, -(-2 * L2_BYTES // (met * 2 * ff_pad * d * 2)))
    up, down = ([random_bf16(ctx, n * r * c, i) for i in range(copies)] for r, c in ((2 * ff_pad, d), (d, ff_pad)))
    rows = max(slots, 32) + 256
    x, a, y = random_bf16(ctx, rows * d, 5), random_bf16(ctx, rows * ff_pad, 6), ctx.alloc(rows * d * 2)
    ms1 = time_graph(lambda i, s: ctx.plain_gemm_experts(BF16, up[i % copies], n, 2 * ff_pad, d, x, d, rows, not tensor, lists, slots, few, tensor, True, a, ff_pad, ff_pad,
                                                         stream=s), iters)
    ms2 = time_graph(lambda i, s: ctx.plain_gemm_experts(BF16, down[i % copies], n, d, ff_pad, a, ff_pad, rows, False, lists, slots, few, tensor, False, y, d, d,
                                                         stream=s), iters)
    for b in [logits, corr, x, a, y] + up + down:
        b.free()
    lists.free()
    out = [dict(peaks.entry("choice of experts, lists", route, tokens * n * 4.0 + slots * 16.0), tokens=tokens),
           dict(peaks.entry("experts' gate|up pairs", ms1, 2.0 * met * 2 * ff * d + 2.0 * slots * (d + ff), 4.0 * ff * d * slots), tokens=tokens, experts_met=met),
           dict(peaks.entry("experts' down", ms2, 2.0 * met * ff * d + 2.0 * slots * (d + ff), 2.0 * ff * d * slots), tokens=tokens, experts_met=met)]
    return out


def kernels(ctx, peaks, shape, iters):
    sh = SHAPES[shape]
    d, (nq, nkv, hd) = sh["d"], sh["attention"]
    sd, (sh_, sv, sn, sg) = latentbench.SHAPES[shape], sh["ssd"]
    window = plainbench.SHAPES[shape][5]
    up = lambda n: (n + 127) // 128 * 128
    inner = sh_ * sv
    in_rows = {"parallel": 2 * nq * hd + 2 * nkv * hd + 2 * inner + 2 * sg * sn + sh_, "HGRN2": sh["forget"][0] * (2 * sh["forget"][1] + sh["forget"][2]),
               "mLSTM": sh["mlstm"][0] * (2 * sh["mlstm"][1] + 2 * sh["mlstm"][2] + 2)}
    mm = []
    for t in (1, 8, 64, 128, 2048):
        it = iters if t <= 128 else max(4, iters // 4)
        mm += [plain_matmul(ctx, peaks, "input of %s" % k, up(n), d, t, "store", it) for k, n in in_rows.items()]
        mm += [plain_matmul(ctx, peaks, "o|o", d, nq * hd + inner, t, "store", it)]
        mm += experts(ctx, peaks, d, sh["experts"], t, it)
        mm += [plain_matmul(ctx, peaks, "Gimozen q|k|v", (nq + 2 * nkv) * hd, d, t, "store", it), plain_matmul(ctx, peaks, "Gimozen gate|up pairs", 2 * sd["ff"], d, t, "pairs", it),
               plain_matmul(ctx, peaks, "Gimozen down + scaled residual", d, sd["ff"], t, "add", it)]
    att = []
    for streams, rows in ((1, 1), (8, 1), (64, 1), (1, 6), (64, 6), (1, 128), (1, 2048)):
        it = iters if rows < 2048 else max(4, iters // 4)
        att += [attention(ctx, peaks, "chunked attention", nq, nkv, hd, window, rows, streams, it),
                latentbench.value_attention(ctx, peaks, "Gimozen attention", nq, nkv, hd, hd, window, rows, streams, it)]
    rec = []
    for streams, rows in ((1, 1), (8, 1), (64, 1), (8, 6), (1, 128), (1, 2048), (8, 512)):
        it = iters if rows < 128 else max(4, iters // 4)
        rec += [recurrence(ctx, peaks, REC_FORGET, *sh["forget"], rows, streams, it), recurrence(ctx, peaks, REC_MLSTM, *sh["mlstm"], rows, streams, it),
                recurrence(ctx, peaks, REC_SSD, sh_, sn, sv, rows, streams, it, groups=sg)]
    norms = []
    for rows in (1, 64, 2048):
        norms += [output_norm(ctx, peaks, "output norm + convolution", d, sh["norm_groups"], rows, iters),
                  projection_norms(ctx, peaks, "projection norms", nq, nkv, hd, rows, iters), short_conv(ctx, peaks, "short convolution", inner + 2 * sg * sn, rows, iters),
                  gated_norm(ctx, peaks, "gated norm", inner, sg, rows, iters), latentbench.post_norm(ctx, peaks, "Gimozen post norm", d, rows, iters),
                  latentbench.head_norms(ctx, peaks, "Gimozen query and key norms", nq, nkv, hd, nkv, hd, hd, rows, iters)]
    return {"matmuls": mm, "attention": att, "recurrences": rec, "norms": norms}


# ------------------------------------------------------------------ whole models
def layer_list(shape):
    """Parallel, HGRN2, parallel, mLSTM, over and over."""
    sh = SHAPES[shape]
    (nq, nkv, hd), (h, v, n, g) = sh["attention"], sh["ssd"]
    e, top, ff, groups, keep = sh["experts"]
    moe = dict(ffn=ff, act=SILU, experts=e, expert_top=top, expert_groups=groups, expert_keep=keep)
    rec = lambda kind, s, **kw: PlainLayer(recurrence=kind, rec_heads=s[0], rec_dim=s[1], rec_vdim=s[2], **kw, **moe)
    parallel = PlainLayer(n_q_heads=nq, n_kv_heads=nkv, head_dim=hd, value_dim=hd, score_scale=hd ** -0.5, chunk=CHUNK, qk_norm=NORM_PROJECTION, qkv_bias=1, linear_bias=1,
                          sink=1, value_gate=1, attn_scale=0.5, rec_scale=0.5, recurrence=REC_SSD, rec_heads=h, rec_dim=n, rec_vdim=v, rec_groups=g, rec_taps=TAPS,
                          rec_norm_groups=g, **moe)
    cycle = [parallel, rec(REC_FORGET, sh["forget"]), parallel, rec(REC_MLSTM, sh["mlstm"], rec_cap=15.0)]
    return [cycle[i % 4] for i in range(sh["layers"])]


def tarivik_model(ctx, shape, max_context):
    sh = SHAPES[shape]
    layers = layer_list(shape)
    m = PlainModel(ctx, PlainConfig(n_layers=len(layers), d_model=sh["d"], vocab=sh["vocab"], max_context=max_context, compute=BF16, norm_eps=1e-6, output_norm=1,
                                    norm_groups=sh["norm_groups"], conv_taps=TAPS, positions=max_context), layers)
    m.fill(seed=1)
    return m


def experts_met(layer, tokens):
    """Experts that at least one of `tokens` tokens meets, choices spread evenly."""
    return layer.experts * (1 - (1 - layer.expert_top / layer.experts) ** tokens)


def pass_bytes(m, streams, context):
    """Matrices, of which every expert that is met counts once; cached rows; states, read and written."""
    n = m.weight_bytes
    for l in m.layers:
        if l.experts:
            n += 2 * 3 * l.ffn * m.cfg.d_model * (experts_met(l, streams) - l.expert_top)
        n += streams * context * 2 * l.n_kv_heads * (l.head_dim + (l.value_dim or 0))
        if l.recurrence:
            n += streams * 2 * 4 * l.rec_heads * l.rec_dim * l.rec_vdim
    return n


def models(ctx, peaks, shape, steps, context=4096):
    out = {}
    vocab = SHAPES[shape]["vocab"]
    for kind, make in (("tarivik", tarivik_model), ("gimozen", latentbench.gimozen_model)):
        m = make(ctx, shape, context + steps + 16)
        res = {"weight_bytes": m.weight_bytes, "decode": [], "prefill": []}
        for streams in (1, 8, 32):
            ms = decode(ctx, m, streams, context, steps)
            nbytes = pass_bytes(m, streams, context) if kind == "tarivik" else m.weight_bytes + streams * context * latentbench.cache_row_bytes(m.layers)
            res["decode"].append({"streams": streams, "context": context, "ms_per_pass": round(ms, 3), "tokens_per_s": round(streams / ms * 1e3, 1),
                                  "frac": round(nbytes / peaks.hbm / (ms * 1e-3), 3)})
        for n in (512, 2048):
            prompt = np.random.default_rng(n).integers(0, vocab, size=n).astype(np.int32)
            sess = Session(ctx, m, None, 1, 1, step_rows=n)

            def run():
                sess.step([(0, prompt.tolist(), [n - 1])])
                sess.reset(0)
            ms = on_stream(sess, run, max(3, steps // 4))
            sess.close()
            # the products of every layer (the head runs for one row), the attention of the visible half, the recurrences
            flops = 2.0 * n * (m.weight_bytes / 2 - vocab * m.cfg.d_model)
            flops += sum(2.0 * l.n_q_heads * (l.head_dim + l.rot_dim + (l.value_dim or l.head_dim)) * n * n / 2 for l in m.layers)
            flops += sum(4.0 * n * l.rec_heads * l.rec_dim * l.rec_vdim for l in m.layers)
            t = max(flops / peaks.tf, (pass_bytes(m, n, 0) - sum(8 * (n - 1) * l.rec_heads * l.rec_dim * l.rec_vdim for l in m.layers)) / peaks.hbm)
            res["prefill"].append({"tokens": n, "ms": round(ms, 2), "tokens_per_s": round(n / ms * 1e3, 1), "tflops": round(flops / ms / 1e9, 1),
                                   "frac": round(t / (ms * 1e-3), 3)})
        m.close()
        out[kind] = res
    return out


def run(device, hbm_gbs, bf16_tflops, shapes=("8b", "2b"), steps=12, iters=24, parts=("kernels", "models")):
    ctx = capi.Ctx(device)
    peaks = Peaks(hbm_gbs, bf16_tflops)
    out = {}
    for shape in shapes:
        out[shape] = {"shape": SHAPES[shape]}
        if "kernels" in parts:
            out[shape]["kernels"] = kernels(ctx, peaks, shape, iters)
        if "models" in parts:
            out[shape]["models"] = models(ctx, peaks, shape, steps)
    launches = ctx.launches
    ctx.close()
    return out, launches
