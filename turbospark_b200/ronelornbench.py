"""Prefill and decode throughput of Ronelorn-shaped models beside Gimozen-shaped ones of equal size, and the time of each kernel against
its roofline beside the like kernel (python bench.py --design ronelorn).  Method as in plainbench.
"""
import ctypes as C

import numpy as np

from . import capi, latentbench, plainbench, tarivikbench
from .model import Session
from .plain import (BF16, NORM_HEAD, NORM_PROJECTION, REC_FORGET, REC_MINGRU, RELU2, SINK_ZERO, PlainConfig, PlainLayer, PlainModel)
from .plainbench import L2_BYTES, Peaks, decode, on_stream, plain_matmul, random_bf16, time_graph

# Equal to latentbench's shapes in width, attention heads, layers and vocabulary; two matrices of 3/2 the width hold as much as a gated feed-forward's three,
# and four of `scan` channels as much as the attention's.
SHAPES = {"8b": dict(d=4096, layers=32, vocab=128256, ff=21504, attention=(32, 8, 128), window=2048, scan=2560),
          "2b": dict(d=2048, layers=16, vocab=128256, ff=12288, attention=(32, 8, 64), window=1024, scan=1280)}
KEEP, POOL, RING = 64, 16, 8
CONTEXT = 8192  # of the attention kernels


def seen(context, rows, window, kind):
    """Rows of the cache that the queries at positions context .. see, summed, and the distinct ones."""
    def of(p):
        before = max(0, p - window + 1)
        return min(p + 1, window), before // POOL if kind == "blocks" else min(KEEP, before) if kind == "kept" else 0
    per = [of(context + r) for r in range(rows)]
    return sum(a + b for a, b in per), min(context + rows, window + rows - 1) + per[-1][1]


def attention(ctx, peaks, name, kind, nq, nkv, hd, context, rows, streams, window, iters):
    pages = (context + rows + 63) // 64 + 1
    total, distinct = seen(context, rows, window, kind)
    layers = max(2, -(-2 * L2_BYTES // (streams * distinct * nkv * 2 * hd * 2)))
    kv = capi.PlainCache(ctx, BF16, layers, nkv, hd, hd, 64, pages * streams, streams, pages, pool=POOL if kind == "blocks" else 0)
    for s in range(streams):
        kv.fill_random(s, context + rows, 7 + s)
    n = streams * rows
    q, out, rd = random_bf16(ctx, n * nq * hd, 3, amp=3.5), ctx.alloc(n * nq * hd * 2), latentbench._rows(ctx, context, rows, streams)
    sink, turn, scratch = ctx.zeroed(nq * 4), ctx.to_device(np.tile(np.float32([0.8, 0.6]), n * hd // 2)), ctx.window_attention_scratch()
    extras = dict(blocks=True, cap=30.0, turn=turn, turn_half=hd // 2) if kind == "blocks" else dict(keep=KEEP, sink=sink)
    ms = time_graph(lambda i, s: ctx.plain_attention(kv, i % layers, q, nq * hd, out, nq * hd, rd, [rows] * streams, nq, hd ** -0.5, context + rows, scratch, window=window, stream=s,
                                                     **extras), iters)
    kv.close()
    for b in (q, out, rd, sink, turn, scratch):
        b.free()
    nbytes = streams * distinct * nkv * 2 * hd * 2 + n * nq * 2 * hd * 2 + (n * hd * 4 if kind == "blocks" else 0)
    return dict(peaks.entry(name, ms, nbytes, 4.0 * hd * nq * total * streams), context=context, rows=rows, streams=streams, window=window)


def scan(ctx, peaks, name, width, rows, streams, iters):
    n = streams * rows
    copies = min(64, max(2, -(-2 * L2_BYTES // (n * width * 12))))
    gate = [ctx.to_device(np.random.default_rng(i).standard_normal(n * 2 * width).astype(np.float32)) for i in range(copies)]
    g, out = random_bf16(ctx, copies * n * width, 1, amp=2.0), ctx.alloc(copies * n * width * 2)
    state, rd = ctx.zeroed(streams * 2 * width * 4), latentbench._rows(ctx, 0 if rows >= 64 else 4096, rows, streams)
    sums = ctx.zeroed(streams * (rows // 128 + 1) * width * 8)

    def call(i, s):
        at = (i % copies) * n * width * 2
        ctx.gated_scan_rows(BF16, gate[i % copies], 2 * width, C.c_void_p(g.ptr + at), width, width, state, streams, 2, rd, n, rows, C.c_void_p(out.ptr + at), width, chunked=rows >= 64, sums=sums, stream=s)
    ms = time_graph(call, iters)
    for b in gate + [g, out, state, rd, sums]:
        b.free()
    return dict(peaks.entry(name, ms, n * width * 12.0 + streams * width * 8.0), rows=rows, streams=streams, width=width)


def feed_forward(ctx, peaks, name, rows, cols, tokens, kind, iters):
    """up: an activation behind the product, stored in the compute type; down: scaled sums added to the stream."""
    copies = max(2, -(-2 * L2_BYTES // (rows * cols * 2)))
    ws = [random_bf16(ctx, rows * cols, i) for i in range(copies)]
    x_rows = max(32, tokens)
    x, work, y = random_bf16(ctx, x_rows * cols, 9), ctx.plain_gemm_workspace(), ctx.zeroed(tokens * rows * 4)
    if kind == "up":
        ms = time_graph(lambda i, s: ctx.plain_gemm_act(BF16, ws[i % copies], rows, cols, x, x_rows, tokens, y, rows, rows, RELU2, work, stream=s), iters)
    else:
        ms = time_graph(lambda i, s: ctx.plain_gemm_add(BF16, ws[i % copies], rows, cols, x, x_rows, tokens, y, rows, rows, 1.0, 0.7, work, stream=s), iters)
    for b in ws + [x, work, y]:
        b.free()
    return dict(peaks.entry(name, ms, 2 * cols * (rows + tokens) + tokens * rows * (2 if kind == "up" else 8), 2.0 * rows * cols * tokens), rows=rows, cols=cols, tokens=tokens)


def pre_norm(ctx, peaks, name, d, rows, iters):
    copies = max(2, -(-2 * L2_BYTES // (rows * d * 6))) if rows > 256 else 2
    xs, outs, w = [ctx.zeroed(rows * d * 4) for _ in range(copies)], [ctx.alloc(rows * d * 2) for _ in range(copies)], ctx.zeroed(d * 4)
    ms = time_graph(lambda i, s: ctx.pre_norm_rows(BF16, xs[i % copies], d, w, 1e-6, rows, outs[i % copies], d, stream=s), iters)
    for b in xs + outs + [w]:
        b.free()
    return dict(peaks.entry(name, ms, rows * d * 6.0), rows=rows, d=d)


def turned_norms(ctx, peaks, name, nq, nk, hd, projection, rows, iters):
    kv, layers = latentbench._cache(ctx, nk, hd, hd, 0, rows, 1)
    nv = 0 if projection else nk
    per = (nq + nk + nv) * hd
    copies = max(2, -(-2 * L2_BYTES // (rows * per * 6))) if rows > 256 else 2
    raws, qs = [ctx.zeroed(rows * per * 4) for _ in range(copies)], [ctx.alloc(rows * nq * hd * 2) for _ in range(copies)]
    w, table, rd = ctx.zeroed(nq * hd * 4), ctx.zeroed(rows * hd * 4), latentbench._rows(ctx, 0, rows, 1)
    ms = time_graph(lambda i, s: ctx.turned_norm_rows(kv, i % layers, raws[i % copies], per, nq, nk, hd, w, w, 1e-6, rd, rows, qs[i % copies], nq * hd, rot=table, rot_half=hd // 2,
                                                      n_v=nv, v_width=hd, turn=None if projection else table, turn_half=hd // 2, projection=projection, stream=s), iters)
    kv.close()
    for b in raws + qs + [w, table, rd]:
        b.free()
    return dict(peaks.entry(name, ms, rows * per * 6.0), rows=rows)


def block_means(ctx, peaks, name, nk, hd, rows, streams, iters):
    pages = (rows + 4096 + 63) // 64 + 1
    layers = max(2, -(-2 * L2_BYTES // (streams * rows * nk * 2 * hd * 2)) if rows > 256 else 2)
    kv = capi.PlainCache(ctx, BF16, layers, nk, hd, hd, 64, pages * streams, streams, pages, pool=POOL)
    for s in range(streams):
        kv.fill_random(s, 4096 + rows, 7 + s)
    rd = latentbench._rows(ctx, 4095 if rows == 1 else 4096, rows, streams)  # a single row ends a block
    ms = time_graph(lambda i, s: ctx.block_mean_rows(kv, i % layers, rd, streams * rows, stream=s), iters)
    kv.close(), rd.free()
    blocks = streams * max(1, rows // POOL)
    return dict(peaks.entry(name, ms, blocks * (POOL + 1) * nk * 2 * hd * 2.0), rows=rows, streams=streams)


def kernels(ctx, peaks, shape, iters):
    sh, sd = SHAPES[shape], latentbench.SHAPES[shape]
    d, (nq, nkv, hd), window = sh["d"], sh["attention"], sh["window"]
    mm = []
    for t in (1, 8, 64, 128, 2048):
        it = iters if t <= 128 else max(4, iters // 4)
        mm += [plain_matmul(ctx, peaks, "q|k|v", (nq + 2 * nkv) * hd, d, t, "store", it), plain_matmul(ctx, peaks, "g|z|x", 3 * sh["scan"], d, t, "store", it),
               feed_forward(ctx, peaks, "up, squared relu", sh["ff"], d, t, "up", it), feed_forward(ctx, peaks, "down, scaled sum", d, sh["ff"], t, "down", it),
               plain_matmul(ctx, peaks, "Gimozen gate|up pairs", 2 * sd["ff"], d, t, "pairs", it), plain_matmul(ctx, peaks, "Gimozen down + scaled residual", d, sd["ff"], t, "add", it)]
    att = []
    for streams, rows in ((1, 1), (8, 1), (64, 1), (1, 6), (64, 6), (1, 128), (1, 2048)):
        it = iters if rows < 2048 else max(4, iters // 4)
        at = CONTEXT - rows
        att += [attention(ctx, peaks, "window + blocks", "blocks", nq, nkv, hd, at, rows, streams, window, it),
                attention(ctx, peaks, "window + kept tokens", "kept", nq, nkv, hd, at, rows, streams, window, it),
                latentbench.value_attention(ctx, peaks, "Gimozen attention", nq, nkv, hd, hd, window, rows, streams, it)]
    rec = []
    for streams, rows in ((1, 1), (8, 1), (64, 1), (8, 6), (1, 128), (1, 2048), (8, 512)):
        it = iters if rows < 128 else max(4, iters // 4)
        rec += [scan(ctx, peaks, "minGRU", sh["scan"], rows, streams, it),
                tarivikbench.recurrence(ctx, peaks, REC_FORGET, *tarivikbench.SHAPES[shape]["forget"], rows, streams, it)]
    norms = []
    for rows in (1, 64, 2048):
        norms += [pre_norm(ctx, peaks, "pre-norm", d, rows, iters), turned_norms(ctx, peaks, "head norms, rotations, turned values", nq, nkv, hd, False, rows, iters),
                  turned_norms(ctx, peaks, "projection norms, rotations", nq, nkv, hd, True, rows, iters), block_means(ctx, peaks, "block means", nkv, hd, rows, 1, iters),
                  latentbench.post_norm(ctx, peaks, "Gimozen post norm", d, rows, iters),
                  latentbench.head_norms(ctx, peaks, "Gimozen query and key norms", nq, nkv, hd, nkv, hd, hd, rows, iters),
                  tarivikbench.projection_norms(ctx, peaks, "Tarivik projection norms", nq, nkv, hd, rows, iters)]
    return {"matmuls": mm, "attention": att, "recurrences": rec, "norms": norms}


# ------------------------------------------------------------------ whole models
def layer_list(shape):
    """Kept tokens, minGRU, blocks, over and over."""
    sh = SHAPES[shape]
    nq, nkv, hd = sh["attention"]
    ff = dict(ffn=sh["ff"], act=RELU2, ff_plain=1)
    heads = dict(n_q_heads=nq, n_kv_heads=nkv, head_dim=hd, value_dim=hd, score_scale=hd ** -0.5, window=sh["window"], rot_dim=hd, rot_base=5e5, **ff)
    cycle = [PlainLayer(qk_norm=NORM_PROJECTION, sink=SINK_ZERO, keep_first=KEEP, **heads), PlainLayer(recurrence=REC_MINGRU, rec_heads=1, rec_dim=1, rec_vdim=sh["scan"], **ff),
             PlainLayer(qk_norm=NORM_HEAD, value_rot=1, pool=POOL, score_cap=30.0, rot_factor=4.0, **heads)]
    return [cycle[i % 3] for i in range(sh["layers"])]


def ronelorn_model(ctx, shape, max_context):
    sh, layers = SHAPES[shape], layer_list(shape)
    m = PlainModel(ctx, PlainConfig(n_layers=len(layers), d_model=sh["d"], vocab=sh["vocab"], max_context=max_context, compute=BF16, norm_eps=1e-6, pre_norm=1, sublayer_scale=0.7),
                   layers)
    m.fill(seed=1)
    return m


def pass_bytes(m, streams, context):
    """Matrices; cached rows and blocks that a token sees; states, read and written."""
    n = m.weight_bytes
    for l in m.layers:
        if l.n_q_heads:
            n += streams * seen(context, 1, l.window, "blocks" if l.pool else "kept")[0] * 2 * l.n_kv_heads * 2 * l.head_dim
        n += streams * 8 * l.rec_vdim
    return n


def models(ctx, peaks, shape, steps, context=4096):
    out, vocab = {}, SHAPES[shape]["vocab"]
    for kind, make in (("ronelorn", ronelorn_model), ("gimozen", latentbench.gimozen_model)):
        m = make(ctx, shape, context + steps + 16)
        res = {"weight_bytes": m.weight_bytes, "decode": [], "prefill": []}
        for streams in (1, 8, 32):
            ms = decode(ctx, m, streams, context, steps)
            nbytes = pass_bytes(m, streams, context) if kind == "ronelorn" else m.weight_bytes + streams * context * latentbench.cache_row_bytes(m.layers)
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
            # the products of every layer (the head runs for one row) and the attention of what is visible
            flops = 2.0 * n * (m.weight_bytes / 2 - vocab * m.cfg.d_model)
            flops += sum(2.0 * l.n_q_heads * (l.head_dim + (0 if kind == "ronelorn" else l.rot_dim) + (l.value_dim or l.head_dim)) *
                         (seen(0, n, l.window, "blocks" if l.pool else "kept")[0] if l.window else n * n / 2) for l in m.layers if l.n_q_heads)
            t = max(flops / peaks.tf, m.weight_bytes / peaks.hbm)
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
