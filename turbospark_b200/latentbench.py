"""Prefill and decode throughput of Gimozen-shaped models beside Nigenex-shaped ones of equal size, and the time of each kernel
against its roofline beside the like kernel (python bench.py --design gimozen).  Method as in plainbench.
"""
import ctypes as C

import numpy as np

from . import capi, plainbench
from .model import Session
from .plain import BF16, SILU, PlainConfig, PlainLayer, PlainModel
from .plainbench import L2_BYTES, Peaks, decode, on_stream, plain_matmul, random_bf16, time_graph, visible, window_attention

# d, feed-forward, layers, vocabulary; latent layers: heads, plain, rotated and value columns of a head, latent;
# attention layers: query heads, key heads, head size.  Equal in width, heads, feed-forward, layers and vocabulary to plainbench's shapes.
SHAPES = {"8b": dict(d=4096, ff=14336, layers=32, vocab=128256, latent=(32, 128, 64, 128, 512), attention=(32, 8, 128)),
          "2b": dict(d=2048, ff=8192, layers=16, vocab=128256, latent=(32, 64, 32, 64, 256), attention=(32, 8, 64))}


def _rows(ctx, context, rows, streams):
    return ctx.to_device(capi.row_descs([(s, context, j, context + j, 0) for s in range(streams) for j in range(rows)]))


def _cache(ctx, kv_heads, key_dim, value_dim, context, rows, streams):
    pages = (context + rows + 63) // 64 + 1
    layers = max(2, -(-2 * L2_BYTES // (streams * (context + rows) * kv_heads * (key_dim + value_dim) * 2)))
    kv = capi.PlainCache(ctx, BF16, layers, kv_heads, key_dim, value_dim, 64, pages * streams, streams, pages)
    for s in range(streams):
        kv.fill_random(s, context + rows, 7 + s)
    return kv, layers


def value_attention(ctx, peaks, name, nq, nkv, kd, vd, context, rows, streams, iters, sink=False, gated=False):
    """Keys and values of their own; kd != vd: the expanded form of a latent layer."""
    kv, layers = _cache(ctx, nkv, kd, vd, context, rows, streams)
    n = streams * rows
    q, out, rd = random_bf16(ctx, n * nq * kd, 3, amp=3.5), ctx.alloc(n * nq * vd * 2), _rows(ctx, context, rows, streams)
    extras = {}
    if sink:
        extras["sink"] = ctx.zeroed(nq * 4)
    if gated:
        extras.update(value_gate=random_bf16(ctx, n * nq * vd, 4), value_gate_stride=nq * vd)
    scratch = ctx.window_attention_scratch()
    ms = time_graph(lambda i, s: ctx.plain_attention(kv, i % layers, q, nq * kd, out, nq * vd, rd, [rows] * streams, nq, kd ** -0.5, context + rows, scratch,
                                                     stream=s, **extras), iters)
    seen, distinct = visible(context, rows, 0)
    kv.close()
    for b in [q, out, rd, scratch] + [v for v in extras.values() if not isinstance(v, int)]:
        b.free()
    nbytes = streams * distinct * nkv * (kd + vd) * 2 + n * nq * (kd + vd * (2 if gated else 1)) * 2
    return dict(peaks.entry(name, ms, nbytes, 2.0 * (kd + vd) * nq * seen * streams), context=context, rows=rows, streams=streams)


def latent_attention(ctx, peaks, name, heads, rank, rot, context, rows, streams, iters):
    kv, layers = _cache(ctx, 1, rank + rot, 0, context, rows, streams)
    n, dk = streams * rows, rank + rot
    q, out, rd = random_bf16(ctx, n * heads * dk, 3, amp=3.5), ctx.alloc(n * heads * rank * 2), _rows(ctx, context, rows, streams)
    sink, scratch = ctx.zeroed(heads * 4), ctx.window_attention_scratch()
    ms = time_graph(lambda i, s: ctx.latent_attention(kv, i % layers, q, heads * dk, out, heads * rank, rd, [rows] * streams, heads, rank, dk ** -0.5, sink,
                                                      context + rows, scratch, stream=s), iters)
    seen, distinct = visible(context, rows, 0)
    kv.close()
    for b in (q, out, rd, sink, scratch):
        b.free()
    nbytes = streams * distinct * dk * 2 + n * heads * (dk + rank) * 2
    return dict(peaks.entry(name, ms, nbytes, 2.0 * (dk + rank) * heads * seen * streams), context=context, rows=rows, streams=streams)


def head_matmul(ctx, peaks, name, heads, n_valid, cols, x_step, tokens, gated, iters):
    rows = (n_valid + 127) // 128 * 128
    copies = max(2, -(-2 * L2_BYTES // (heads * rows * cols * 2)))
    ws = [random_bf16(ctx, heads * rows * cols, i) for i in range(copies)]
    x_rows = max(32, tokens)
    x, y, work = random_bf16(ctx, x_rows * heads * x_step, 9), ctx.zeroed(tokens * heads * rows * 2), ctx.plain_gemm_workspace()
    gate = random_bf16(ctx, tokens * heads * n_valid, 5) if gated else None
    ms = time_graph(lambda i, s: ctx.plain_gemm_heads(BF16, ws[i % copies], heads, rows, cols, x, heads * x_step, x_step, x_rows, tokens, y, heads * rows, rows,
                                                      n_valid, work, gate=gate, gate_stride=heads * n_valid, gate_step=n_valid, stream=s), iters)
    for b in ws + [x, y, work] + ([gate] if gated else []):
        b.free()
    nbytes = 2 * heads * (n_valid * cols + tokens * (cols + n_valid * (2 if gated else 1)))
    return dict(peaks.entry(name, ms, nbytes, 2.0 * heads * n_valid * cols * tokens), rows=heads * n_valid, cols=cols, tokens=tokens)


def post_norm(ctx, peaks, name, d, rows, iters):
    copies = max(2, -(-2 * L2_BYTES // (rows * d * 10))) if rows > 256 else 2
    xs, outs, w = [ctx.zeroed(rows * d * 4) for _ in range(copies)], [ctx.alloc(rows * d * 2) for _ in range(copies)], ctx.zeroed(d * 4)
    ms = time_graph(lambda i, s: ctx.post_norm_rows(BF16, xs[i % copies], d, w, 1e-6, rows, outs[i % copies], d, stream=s), iters)
    for b in xs + outs + [w]:
        b.free()
    return dict(peaks.entry(name, ms, rows * d * 10.0), rows=rows, d=d)


def head_norms(ctx, peaks, name, nq, nk, width, kv_heads, key_dim, value_dim, rows, iters):
    kv, layers = _cache(ctx, kv_heads, key_dim, value_dim, 0, rows, 1)
    per = (nq + nk) * width
    copies = max(2, -(-2 * L2_BYTES // (rows * per * 6))) if rows > 256 else 2
    raws, qs = [ctx.zeroed(rows * per * 4) for _ in range(copies)], [ctx.alloc(rows * max(nq, 1) * key_dim * 2) for _ in range(copies)]
    w, rd = ctx.zeroed(width * 4), _rows(ctx, 0, rows, 1)
    ms = time_graph(lambda i, s: ctx.head_norm_rows(kv, i % layers, raws[i % copies], per, nq, nk, width, w, w, 1e-6, rd, rows, qs[i % copies],
                                                    max(nq, 1) * key_dim, temp_coef=0.3 if nq else 0.0, temp_every=512 if nq else 0, stream=s), iters)
    kv.close()
    for b in raws + qs + [w, rd]:
        b.free()
    return dict(peaks.entry(name, ms, rows * per * 6.0), rows=rows, width=width)


def kernels(ctx, peaks, shape, iters):
    sh = SHAPES[shape]
    d, ff = sh["d"], sh["ff"]
    H, D, R, E, K = sh["latent"]
    nq, nkv, hd = sh["attention"]
    _, _, _, _, _, window, _, _ = plainbench.SHAPES[shape]
    mm = []
    for t in (1, 8, 64, 128, 2048):
        it = iters if t <= 128 else max(4, iters // 4)
        up = lambda n: (n + 127) // 128 * 128
        mm += [plain_matmul(ctx, peaks, "q|k|v", (nq + 2 * nkv) * hd, d, t, "store", it),
               plain_matmul(ctx, peaks, "q|latent|gates|rotated", up(H * (D + R) + K + R + H * E), d, t, "store", it),
               plain_matmul(ctx, peaks, "o + scaled residual", d, H * E, t, "add", it), plain_matmul(ctx, peaks, "gate|up pairs", 2 * ff, d, t, "pairs", it),
               plain_matmul(ctx, peaks, "down + scaled residual", d, ff, t, "add", it)]
        if t <= 128:
            mm += [head_matmul(ctx, peaks, "absorb", H, K, D, (D + R + 63) // 64 * 64, t, False, it), head_matmul(ctx, peaks, "lift, gated", H, E, K, K, t, True, it)]
        else:
            mm.append(plain_matmul(ctx, peaks, "expand", H * (D + E), K, t, "store", it))
        mm.append(plain_matmul(ctx, peaks, "Nigenex queries|keys|gates", (nq * hd + nkv * hd + nq + 127) // 128 * 128, d, t, "store", it))
        mm.append(plain_matmul(ctx, peaks, "Nigenex [o|down] + residual", d, nq * hd + ff, t, "add", it))
    att = []
    ctx_len = 8192 if window >= 4096 else 4096
    for streams, rows in ((1, 1), (8, 1), (64, 1), (1, 6), (64, 6), (1, 32), (1, 128), (1, 2048)):
        it = iters if rows < 2048 else max(4, iters // 4)
        att.append(value_attention(ctx, peaks, "attention, keys and values", nq, nkv, hd, hd, window, rows, streams, it))
        if rows < 64:
            att.append(latent_attention(ctx, peaks, "latent attention", H, K, R, window, rows, streams, it))
        else:
            att.append(value_attention(ctx, peaks, "latent attention, expanded", H, H, (D + R + 63) // 64 * 64, E, 0 if rows == 2048 else window, rows, streams, it,
                                       sink=True, gated=True))
        # over as many keys: a full window
        att.append(window_attention(ctx, peaks, "Nigenex window attention", hd, nq, nkv, ctx_len, rows, streams, window, it))
    norms = []
    for rows in (1, 64, 2048):
        norms += [post_norm(ctx, peaks, "post norm", d, rows, iters), head_norms(ctx, peaks, "query and key norms", nq, nkv, hd, nkv, hd, hd, rows, iters),
                  head_norms(ctx, peaks, "latent norm", 0, 1, K, 1, K + R, 0, rows, iters),
                  plainbench.norm_shift(ctx, peaks, "Nigenex norm + token shift", d, rows, iters)]
    return {"matmuls": mm, "attention": att, "norms": norms}


# ------------------------------------------------------------------ whole models
def layer_list(shape):
    """Latent layers and attention layers in turn; every other latent layer reads the one before it."""
    sh = SHAPES[shape]
    H, D, R, E, K = sh["latent"]
    nq, nkv, hd = sh["attention"]
    rot = dict(rot_dim=R, rot_base=5e5, rot_factor=4.0, rot_original=8192, rot_fast=32, rot_slow=1)
    out = []
    for i in range(sh["layers"]):
        if i % 2:
            out.append(PlainLayer(n_q_heads=nq, n_kv_heads=nkv, head_dim=hd, value_dim=hd, score_scale=hd ** -0.5, qk_norm=1, q_temp_every=4096, q_temp_coef=0.1,
                                  ffn=sh["ff"], act=SILU))
        else:
            out.append(PlainLayer(n_q_heads=H, n_kv_heads=1, head_dim=D, value_dim=E, kv_rank=K, score_scale=(D + R) ** -0.5, sink=1, value_gate=1, ffn=sh["ff"],
                                  act=SILU, kv_source=i - 1 if i % 4 == 2 else 0, **rot))
    return out


def gimozen_model(ctx, shape, max_context):
    sh = SHAPES[shape]
    layers = layer_list(shape)
    m = PlainModel(ctx, PlainConfig(n_layers=len(layers), d_model=sh["d"], vocab=sh["vocab"], max_context=max_context, compute=BF16, norm_eps=1e-6, post_norm=1,
                                    residual_scale=2.0, embed_scale=1.0), layers)
    m.fill(seed=1)
    return m


def cache_row_bytes(layers):
    return sum(2 * ((l.kv_rank + l.rot_dim) if l.kv_rank else l.n_kv_heads * (l.head_dim + (l.value_dim or 0))) for l in layers)


def models(ctx, peaks, shape, steps, context=4096):
    out = {}
    vocab = SHAPES[shape]["vocab"]
    for kind, make in (("gimozen", gimozen_model), ("nigenex", plainbench.plain_model)):
        m = make(ctx, shape, context + steps + 16)
        res = {"weight_bytes": m.weight_bytes, "decode": [], "prefill": []}
        row = cache_row_bytes(m.layers)
        for streams in (1, 8, 32):
            ms = decode(ctx, m, streams, context, steps)
            seen = min(context, m.layers[0].window or context)
            res["decode"].append({"streams": streams, "context": context, "ms_per_pass": round(ms, 3), "tokens_per_s": round(streams / ms * 1e3, 1),
                                  "frac": round((m.weight_bytes + streams * seen * row) / peaks.hbm / (ms * 1e-3), 3)})
        for n in (512, 2048):
            prompt = np.random.default_rng(n).integers(0, vocab, size=n).astype(np.int32)
            sess = Session(ctx, m, None, 1, 1, step_rows=n)

            def run():
                sess.step([(0, prompt.tolist(), [n - 1])])
                sess.reset(0)
            ms = on_stream(sess, run, max(3, steps // 4))
            sess.close()
            # the products of every layer (the head runs for one row) and the attention of the visible half
            flops = 2.0 * n * (m.weight_bytes / 2 - vocab * m.cfg.d_model)
            flops += sum(2.0 * l.n_q_heads * (l.head_dim + l.rot_dim + (l.value_dim or l.head_dim)) * n * n / 2 for l in m.layers)
            res["prefill"].append({"tokens": n, "ms": round(ms, 2), "tokens_per_s": round(n / ms * 1e3, 1), "tflops": round(flops / ms / 1e9, 1),
                                   "frac": round(flops / peaks.tf / (ms * 1e-3), 3)})
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
