"""Prefill and decode throughput of a Nigenex-shaped plain-weight model beside the block-quantised dense model of equal
size, and the time of each kernel against its roofline (python bench.py --design nigenex).

Random weights, random keys.  Device times by CUDA events around launches replayed from a CUDA graph, best of several
repeats after warm-up; every kernel rotates over more than an L2's worth of distinct weights or cache layers.
"""
import ctypes as C

import numpy as np

from . import capi, opbench
from .model import Model, ModelConfig, Session, run_config
from .plain import BF16, GELU_TANH, PlainConfig, PlainLayer, PlainModel

L2_BYTES = opbench.L2_BYTES
# layer shapes: d, query heads, key heads, head size, feed-forward, window, layers, vocabulary
SHAPES = {"8b": (4096, 32, 8, 128, 14336, 4096, 32, 128256), "2b": (2048, 32, 8, 64, 8192, 1024, 16, 128256)}


def time_graph(fn, iters, repeats=5, warm=3):
    """Milliseconds of one call of fn(i, stream), calls 0 .. iters - 1 captured once and replayed."""
    import torch
    side = torch.cuda.Stream()
    ptr = C.c_void_p(side.cuda_stream)
    fn(0, ptr)  # one-time set-up (attributes, tensor maps) outside the capture
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, stream=side):
        for i in range(iters):
            fn(i, ptr)
    best = None
    for r in range(warm + repeats):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record(side)
        with torch.cuda.stream(side):
            g.replay()
        e1.record(side)
        torch.cuda.synchronize()
        if r >= warm:
            ms = e0.elapsed_time(e1) / iters
            best = ms if best is None else min(best, ms)
    return best


class Peaks:
    def __init__(self, hbm_gbs, bf16_tflops):
        self.hbm, self.tf = hbm_gbs * 1e9, bf16_tflops * 1e12

    def entry(self, name, ms, nbytes, flops=0.0):
        """A kernel's line: its roofline time is the slower of its bytes and its flops at the measured peaks."""
        t_mem, t_mma = nbytes / self.hbm, flops / self.tf
        return {"kernel": name, "us": round(ms * 1e3, 2), "bound": "hbm" if t_mem >= t_mma else "tensor", "gbs": round(nbytes / ms / 1e6, 1),
                "tflops": round(flops / ms / 1e9, 1), "frac": round(max(t_mem, t_mma) / (ms * 1e-3), 3)}


# ------------------------------------------------------------------ kernels
def random_bf16(ctx, n, seed, amp=0.05):
    import torch
    torch.manual_seed(seed)
    b = ctx.alloc(n * 2)
    t = torch.empty(min(n, 1 << 22), device="cuda", dtype=torch.bfloat16).uniform_(-amp, amp).view(torch.int16).cpu().numpy()
    for at in range(0, n, t.size):
        m = min(t.size, n - at)
        ctx.check(capi.lib().tsb_memcpy_h2d(ctx.h, None, C.c_void_p(b.ptr + at * 2), t.ctypes.data_as(C.c_void_p), C.c_size_t(m * 2)))
    ctx.sync()
    return b


def plain_matmul(ctx, peaks, name, rows, cols, tokens, kind, iters):
    copies = max(2, -(-2 * L2_BYTES // (rows * cols * 2)))
    ws = [random_bf16(ctx, rows * cols, i) for i in range(copies)]
    x_rows = max(32, tokens)
    x, work = random_bf16(ctx, x_rows * cols, 9), ctx.plain_gemm_workspace()
    y = ctx.zeroed(tokens * rows * (2 if kind == "pairs" else 4))
    if kind == "pairs":
        ms = time_graph(lambda i, s: ctx.plain_gemm_pairs(BF16, ws[i % copies], rows, cols, x, x_rows, tokens, y, rows // 2, rows // 2, GELU_TANH, work,
                                                          stream=s), iters)
        out = tokens * rows // 2 * 2
    else:
        ms = time_graph(lambda i, s: ctx.plain_gemm(BF16, ws[i % copies], rows, cols, x, x_rows, tokens, y, rows, rows, work, add=kind == "add", stream=s), iters)
        out = tokens * rows * (8 if kind == "add" else 4)
    for b in ws + [x, work, y]:
        b.free()
    return dict(peaks.entry(name, ms, 2 * cols * (rows + tokens) + out, 2.0 * rows * cols * tokens), rows=rows, cols=cols, tokens=tokens)


def block_matmul(ctx, peaks, name, rows, cols, tokens, iters):
    w_bytes = rows * (cols // 256) * 144
    copies = max(2, -(-2 * L2_BYTES // w_bytes))
    host = opbench.random_blocks("q4k", rows, cols, np.random.default_rng(1))
    ws = [ctx.upload_weights(host) for _ in range(copies)]
    x = ctx.to_device(opbench.f16_bits(np.random.default_rng(2).standard_normal((tokens, cols))))
    y, work = ctx.alloc(tokens * rows * 2), ctx.alloc(ctx.gemm_workspace_bytes(0, rows, cols, tokens))
    ctx.gemm_prepare(0, rows, cols, x, tokens, work)
    ms = opbench.time_launches(lambda i: ctx.gemm_quant_prepared(0, ws[i % copies], rows, cols, x, work, y, tokens), iters)
    for b in ws + [x, y, work]:
        b.free()
    return dict(peaks.entry(name, ms, w_bytes + 2 * tokens * (rows + cols), 2.0 * rows * cols * tokens), rows=rows, cols=cols, tokens=tokens)


def visible(context, rows, window):
    """Keys that the rows at positions context .. see, summed, and the distinct ones."""
    per_row = [min(context + r + 1, window or 1 << 60) for r in range(rows)]
    return sum(per_row), min(context + rows, (window or 1 << 60) + rows - 1)


def window_attention(ctx, peaks, name, hd, nq, nkv, context, rows, streams, window, iters):
    pages = (context + rows + 63) // 64 + 1
    layers = max(2, -(-2 * L2_BYTES // (streams * min(context + rows, window + rows) * nkv * hd * 2)))
    kv = capi.KeyCache(ctx, BF16, layers, nkv, hd, 64, pages * streams, streams, pages)
    for s in range(streams):
        kv.fill_random(s, context + rows, 7 + s)
    n = streams * rows
    q, out = random_bf16(ctx, n * nq * hd, 3, amp=3.5), ctx.alloc(n * nq * hd * 2)  # scores of standard deviation about 2
    gate = ctx.zeroed(n * nq * 4)
    r1, r2 = ctx.to_device(np.full(nq, 0.7, dtype=np.float32)), ctx.to_device(np.full(nq, 0.2, dtype=np.float32))
    rd = ctx.to_device(capi.row_descs([(s, context, j, context + j, 0) for s in range(streams) for j in range(rows)]))
    scratch = ctx.window_attention_scratch()
    ms = time_graph(lambda i, s: ctx.window_attention(kv, i % layers, q, nq * hd, out, nq * hd, rd, [rows] * streams, nq, hd ** -0.5, 50.0, r1, r2, gate,
                                                      window, context + rows, scratch, stream=s), iters)
    seen, distinct = visible(context, rows, window)
    kv.close()
    for b in (q, out, gate, r1, r2, rd, scratch):
        b.free()
    nbytes = streams * distinct * nkv * hd * 2 + n * nq * hd * 4
    return dict(peaks.entry(name, ms, nbytes, 4.0 * hd * nq * seen * streams), context=context, rows=rows, streams=streams, window=window)


def block_attention(ctx, peaks, name, hd, nq, nkv, context, rows, streams, iters):
    r = opbench.bench_attention(ctx, hd, nq, nkv, context, rows, streams, iters)
    seen = sum(context + j + 1 for j in range(rows))
    return dict(peaks.entry(name, r["us"] * 1e-3, r["bytes"], 4.0 * hd * nq * seen * streams), context=context, rows=rows, streams=streams)


def norm_shift(ctx, peaks, name, d, rows, iters):
    copies = max(2, -(-2 * L2_BYTES // (rows * d * 8))) if rows > 256 else 2
    xs = [ctx.zeroed(rows * d * 4) for _ in range(copies)]
    mixes, hs = [ctx.alloc(rows * d * 2) for _ in range(copies)], [ctx.alloc(rows * d * 2) for _ in range(copies)]
    ring = 4
    streams = rows if rows <= 64 else 1
    per = rows // streams
    rd = ctx.to_device(capi.row_descs([(s, 64, j, 64 + j, 0) for s in range(streams) for j in range(per)]))
    state, gain, mu = ctx.zeroed(streams * ring * d * 4), ctx.to_device(np.ones(1, dtype=np.float32)), ctx.to_device(np.full(d, 0.5, dtype=np.float32))
    ms = time_graph(lambda i, s: ctx.norm_shift_rows(BF16, xs[i % copies], d, gain, 1e-6, mu, rd, rows, state, streams, ring, mixes[i % copies],
                                                     hs[i % copies], d, stream=s), iters)
    for b in xs + mixes + hs + [rd, state, gain, mu]:
        b.free()
    return dict(peaks.entry(name, ms, rows * d * 8.0), rows=rows, d=d)


def block_norm(ctx, peaks, name, d, rows, iters):
    copies = max(2, -(-2 * L2_BYTES // (rows * d * 8))) if rows > 256 else 2
    xs, rs, os_ = ([ctx.zeroed(rows * d * 2) for _ in range(copies)] for _ in range(3))
    w = ctx.to_device(np.full(d, 0x3F80, dtype=np.uint16))
    ms = time_graph(lambda i, s: ctx.rmsnorm_rows(xs[i % copies], rs[i % copies], w, os_[i % copies], rows, d, 1e-6, stream=s), iters)
    for b in xs + rs + os_ + [w]:
        b.free()
    return dict(peaks.entry(name, ms, rows * d * 8.0), rows=rows, d=d)


def kernels(ctx, peaks, shape, iters):
    d, nq, nkv, hd, ff, window, _, _ = SHAPES[shape]
    qkg = (nq * hd + nkv * hd + nq + 127) // 128 * 128
    lines = []
    for t in (1, 8, 32, 64, 128, 512, 2048):
        it = iters if t <= 128 else max(4, iters // 4)
        lines.append([plain_matmul(ctx, peaks, "queries|keys|gates", qkg, d, t, "store", it), plain_matmul(ctx, peaks, "gate|up pairs", 2 * ff, d, t, "pairs", it),
                      plain_matmul(ctx, peaks, "[o|down] + residual", d, nq * hd + ff, t, "add", it)])
        if t <= 128:  # the block-quantised matmuls take 128 rows per pass at most
            lines[-1] += [block_matmul(ctx, peaks, "Q4_K q|k|v", (nq + 2 * nkv) * hd, d, t, it), block_matmul(ctx, peaks, "Q4_K gate|up", 2 * ff, d, t, it),
                          block_matmul(ctx, peaks, "Q4_K down", d, ff, t, it)]
    mm = [e for l in lines for e in l]
    att = []
    ctx_len = 8192 if window >= 4096 else 4096
    for streams, rows in ((1, 1), (8, 1), (64, 1), (1, 6), (64, 6), (1, 128), (1, 2048)):
        it = iters if rows < 2048 else max(4, iters // 4)
        att.append(window_attention(ctx, peaks, "window attention", hd, nq, nkv, ctx_len, rows, streams, window, it))
        if rows <= 128:  # over as many keys as the window holds
            att.append(block_attention(ctx, peaks, "fp16 K/V attention", hd, nq, nkv, window, rows, streams, it))
    norms = []
    for rows in (1, 64, 2048):
        norms += [norm_shift(ctx, peaks, "norm + token shift", d, rows, iters), block_norm(ctx, peaks, "residual + RMSNorm", d, rows, iters)]
    return {"matmuls": mm, "attention": att, "norms": norms}


# ------------------------------------------------------------------ whole models
def plain_model(ctx, shape, max_context):
    d, nq, nkv, hd, ff, window, layers, vocab = SHAPES[shape]
    l = PlainLayer(n_q_heads=nq, n_kv_heads=nkv, head_dim=hd, window=window, score_scale=hd ** -0.5, score_cap=50.0, log_bias=1, head_gate=1,
                   token_shift=1, ffn=ff, act=GELU_TANH)
    m = PlainModel(ctx, PlainConfig(n_layers=layers, d_model=d, vocab=vocab, max_context=max_context, compute=BF16, norm_eps=1e-6, logit_cap=30.0),
                   [l] * layers)
    m.fill(seed=1)
    return m


def block_model(ctx, shape, max_context):
    d, nq, nkv, hd, ff, _, layers, vocab = SHAPES[shape]
    m = Model(ctx, ModelConfig(layers, d, nq, nkv, hd, ff, vocab, max_context, 1e-5, 5e5))
    m.fill_synthetic(capi.Q4_K, seed=1)
    return m


def on_stream(sess, fn, steps, warm=3):
    """Milliseconds per call of fn(), by events on the session's stream."""
    import torch
    st = torch.cuda.ExternalStream(sess.stream_ptr)
    for _ in range(warm):
        fn()
    sess.ctx.sync(C.c_void_p(sess.stream_ptr))
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record(st)
    for _ in range(steps):
        fn()
    e1.record(st)
    sess.ctx.sync(C.c_void_p(sess.stream_ptr))
    return e0.elapsed_time(e1) / steps


def decode(ctx, model, streams, context, steps):
    """One token of every stream per pass, logits left on the device."""
    sess = Session(ctx, model, None, streams, 1)
    sess.fill_context(context, seed=3)
    rng = np.random.default_rng(streams)
    feed = rng.integers(0, model.cfg.vocab, size=(streams, 1)).astype(np.int32)
    ms = on_stream(sess, lambda: sess.verify_tree_streams(feed, [-1], want_logits=False), steps)
    sess.close()
    return ms


def models(ctx, peaks, shape, steps, context=4096):
    d, nq, nkv, hd, ff, window, layers, vocab = SHAPES[shape]
    out = {}
    for kind, make in (("nigenex", plain_model), ("block_q4k", block_model)):
        m = make(ctx, shape, context + steps + 16)
        res = {"weight_bytes": m.weight_bytes, "decode": [], "prefill": []}
        for streams in (1, 8, 32):
            ms = decode(ctx, m, streams, context, steps)
            seen = min(context, window) if kind == "nigenex" else context
            kv = streams * layers * seen * nkv * hd * (2 if kind == "nigenex" else 4)
            res["decode"].append({"streams": streams, "context": context, "ms_per_pass": round(ms, 3), "tokens_per_s": round(streams / ms * 1e3, 1),
                                  "frac": round((m.weight_bytes + kv) / peaks.hbm / (ms * 1e-3), 3)})
        for n in (512, 2048):
            prompt = np.random.default_rng(n).integers(0, vocab, size=n).astype(np.int32)
            if kind == "nigenex":
                sess = Session(ctx, m, None, 1, 1, step_rows=n)

                def run():
                    sess.step([(0, prompt.tolist(), [n - 1])])
                    sess.reset(0)
                ms = on_stream(sess, run, max(3, steps // 4))
            else:
                sess = Session(ctx, m, None, 1, 128)
                rc = run_config(capi.shaping(temperature=0.0), 1, 1)
                ms = min(sess.sequential_run(prompt, rc)[2].prefill_seconds for _ in range(4)) * 1e3
            flops = 2.0 * n * layers * d * (hd * (2 * nq + (nkv if kind == "nigenex" else 2 * nkv)) + 3 * ff)
            res["prefill"].append({"tokens": n, "ms": round(ms, 2), "tokens_per_s": round(n / ms * 1e3, 1), "tflops": round(flops / ms / 1e9, 1),
                                   "frac": round(flops / peaks.tf / (ms * 1e-3), 3)})
            sess.close()
        m.close()
        out[kind] = res
    return out


def run(device, hbm_gbs, bf16_tflops, shapes=("8b", "2b"), steps=12, iters=24, parts=("kernels", "models")):
    ctx = capi.Ctx(device)
    peaks = Peaks(hbm_gbs, bf16_tflops)
    out = {}
    for shape in shapes:
        out[shape] = {"shape": dict(zip(("d", "q_heads", "kv_heads", "head_dim", "ff", "window", "layers", "vocab"), SHAPES[shape]))}
        if "kernels" in parts:
            out[shape]["kernels"] = kernels(ctx, peaks, shape, iters)
        if "models" in parts:
            out[shape]["models"] = models(ctx, peaks, shape, steps)
    launches = ctx.launches
    ctx.close()
    return out, launches
