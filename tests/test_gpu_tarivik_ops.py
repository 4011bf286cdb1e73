"""Output norms with convolutions, projection norms, recurrences, gated norms, routing, grouped products and chunked attention as operators,
against the plain float64 oracle."""
import numpy as np
import pytest

from oracle import tarivik_oracle as to
from tests.test_gpu_gimozen_ops import Cache, f32, padded, upload
from tests.test_gpu_nigenex_ops import descs, fetch, quantise
from turbospark_b200.plain import BF16, F32, REC_FORGET, REC_MLSTM, REC_SSD

pytestmark = pytest.mark.gpu
RELATIVE = {F32: 3e-6, BF16: 9e-3}


@pytest.fixture(scope="module")
def rig():
    import turbospark_b200 as tsb
    ctx = tsb.Ctx(0)
    yield dict(tsb=tsb, ctx=ctx, attn=ctx.window_attention_scratch())
    ctx.close()


def close(got, want, limit):
    """Relative to the rms of what is wanted, per last-but-one index."""
    err = np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())
    assert err.max() < limit, (int(err.argmax()), float(err.max()))


def portions_of(n, sizes):
    out, at = [], 0
    for m in sizes:
        out.append((at, min(m, n - at)))
        at += out[-1][1]
        if at == n:
            break
    assert at == n
    return out


# ------------------------------------------------------------------ end of a sublayer
@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("d,groups,taps,sizes", [(200, 5, 3, [1] * 9 + [2, 7, 30]), (256, 2, 4, [48]), (2048, 4, 4, [1, 1, 46]), (4096, 8, 2, [20, 4]), (5120, 5, 5, [13, 1]),
                                                 (75, 3, 8, [3, 40, 5]), (1001, 7, 2, [20]), (96, 96, 1, [9]), (64, 1, 6, [320, 400])])
def test_output_norm_and_convolution(rig, type_, d, groups, taps, sizes):
    """Two streams in the portions given, the convolution's past carried over."""
    ctx, rng, n, eps = rig["ctx"], np.random.default_rng(d), sum(sizes), 1e-4
    x, y = rng.standard_normal((2, n, d)).astype(np.float32), rng.standard_normal((2, n, d)).astype(np.float32) * rng.uniform(0.1, 3, (2, n, 1)).astype(np.float32)
    w, tw = rng.uniform(0.5, 1.5, d).astype(np.float32), rng.standard_normal((d, taps)).astype(np.float32) * 0.5
    ring, keep = 16, max(taps - 1, 1)
    state, before = ctx.zeroed(2 * ring * d * 4), ctx.zeroed(2 * keep * d * 4)
    wd, td = f32(ctx, w), f32(ctx, tw.T.copy())
    want_x = np.stack([x[s] + to.grouped_rms_norm(y[s].astype(np.float64), w, groups, eps) for s in range(2)])
    want = np.stack([v + to.short_conv(v, tw.astype(np.float64)) for v in want_x])
    stride = (d + 15) // 16 * 16
    for at, m in portions_of(n, sizes):
        if at:  # what a pass copies before a long portion
            past = np.zeros((2, keep, d), dtype=np.float32)
            for k in range(keep):
                if at - keep + k >= 0:
                    past[:, k] = want_x[:, at - keep + k]
            before = f32(ctx, past)
        rows = descs(rig["tsb"], [(s, at, m) for s in range(2)])
        xo, out = ctx.zeroed(2 * m * d * 4), ctx.zeroed(2 * m * stride * 4)
        ctx.output_norm_rows(type_, f32(ctx, x[:, at:at + m].reshape(2 * m, d)), f32(ctx, y[:, at:at + m].reshape(2 * m, d)), d, wd, groups, eps, td, taps, state, 2, ring,
                             ctx.to_device(rows), 2 * m, m, xo, out, stride, before=before)
        close(fetch(xo, F32, (2 * m, d)), want_x[:, at:at + m].reshape(2 * m, d), 2e-6)
        close(fetch(out, type_, (2 * m, stride))[:, :d], want[:, at:at + m].reshape(2 * m, d), RELATIVE[type_])


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("nq,nk,width", [(6, 3, 40), (32, 8, 128), (5, 1, 25), (40, 4, 160)])
def test_projection_norms(rig, type_, nq, nk, width):
    from turbospark_b200.capi import PlainCache
    ctx, rng, n, eps = rig["ctx"], np.random.default_rng(width), 11, 1e-3
    pad = (width + 31) // 32 * 32
    kv = PlainCache(ctx, type_, 1, nk, pad, pad, 16, 4, 2, 2)
    kv.reserve(0, 20), kv.reserve(1, 20)
    raw, wq, wk = rng.standard_normal((2 * n, (nq + nk) * width)).astype(np.float32), rng.uniform(0.5, 1.5, nq * width), rng.uniform(0.5, 1.5, nk * width)
    q = ctx.to_device(np.full(2 * n * nq * pad * 4, 0x7f, dtype=np.uint8))
    ctx.projection_norm_rows(kv, 0, f32(ctx, raw), raw.shape[1], nq, nk, width, f32(ctx, wq), f32(ctx, wk), eps, ctx.to_device(descs(rig["tsb"], [(1, 5, n), (0, 0, n)])),
                             2 * n, q, nq * pad)
    norm = lambda v, w: to.rms(v.astype(np.float64), eps) * w
    got = fetch(q, type_, (2 * n, nq, pad))
    close(got[..., :width].reshape(2 * n, -1), norm(raw[:, :nq * width], wq.astype(np.float32)), RELATIVE[type_])
    assert not got[..., width:].any()
    for s, base, first in ((1, 5, 0), (0, 0, n)):
        rows = kv.read_rows(s, 0, base, n).reshape(n, nk, 2 * pad)[:, :, :width]
        rows = rows.astype(np.float64) if type_ == F32 else (rows.astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        close(rows.reshape(n, -1), norm(raw[first:first + n, nq * width:], wk.astype(np.float32)), RELATIVE[type_])
    kv.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("channels,taps,sizes", [(96, 4, [1, 1, 1, 40, 5]), (77, 3, [2, 20]), (1100, 7, [9, 1, 30]), (32, 1, [5]), (64, 4, [350, 3])])
def test_short_convolution(rig, type_, channels, taps, sizes):
    ctx, rng, n = rig["ctx"], np.random.default_rng(channels), sum(sizes)
    x, u = quantise(rng.standard_normal((n, channels)), type_)
    w, bias = rng.standard_normal((channels, taps)).astype(np.float32) * 0.6, rng.standard_normal(channels).astype(np.float32)
    want = to.silu(to.short_conv(x, w.astype(np.float64), bias.astype(np.float64)))
    ring, keep = 16, max(taps - 1, 1)
    state, wd, bd = ctx.zeroed(ring * channels * 4), f32(ctx, w.T.copy()), f32(ctx, bias)
    stride = (channels + 15) // 16 * 16
    for at, m in portions_of(n, sizes):
        past = np.zeros((keep, channels), dtype=np.float32)
        for k in range(keep):
            if at - keep + k >= 0:
                past[k] = x[at - keep + k]
        out, xp = ctx.zeroed(m * stride * 4), np.zeros((m, stride), dtype=u.dtype)
        xp[:, :channels] = u[at:at + m]
        ctx.short_conv_rows(type_, ctx.to_device(xp), stride, channels, wd, taps, bd, state, 1, ring, ctx.to_device(descs(rig["tsb"], [(0, at, m)])), m, m, out, stride,
                            before=f32(ctx, past))
        close(fetch(out, type_, (m, stride))[:, :channels], want[at:at + m], RELATIVE[type_])


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("width,groups,weight_n,pre,post", [(120, 2, 120, True, False), (165, 5, 33, False, False), (84, 3, 84, False, True), (4096, 8, 4096, True, False),
                                                            (4096, 32, 128, False, True), (20000, 1, 20000, True, False)])
def test_gated_norm(rig, type_, width, groups, weight_n, pre, post):
    ctx, rng, n, eps = rig["ctx"], np.random.default_rng(width), 5, 1e-3
    o, w = rng.standard_normal((n, width)).astype(np.float32), rng.uniform(0.5, 1.5, weight_n).astype(np.float32)
    gate, gu = quantise(rng.standard_normal((n, width)) * 2, type_)
    stride = (width + 15) // 16 * 16
    gp = np.zeros((n, stride), dtype=gu.dtype)
    gp[:, :width] = gu
    g, out = ctx.to_device(gp), ctx.zeroed(n * stride * 4)
    op = np.zeros((n, stride), dtype=np.float32)
    op[:, :width] = o
    ctx.gated_norm_rows(type_, f32(ctx, op), stride, width, groups, f32(ctx, w), weight_n, eps, n, out, stride, scale=0.7, pre_gate=g if pre else None,
                        post_gate=g if post else None, gate_stride=stride if pre or post else 0)
    v = o.astype(np.float64) * (to.silu(gate) if pre else 1.0)
    want = to.grouped_rms_norm(v, np.tile(w, width // weight_n), groups, eps) * (to.sigmoid(gate) if post else 1.0) * 0.7
    close(fetch(out, type_, (n, stride))[:, :width], want, RELATIVE[type_])


# ------------------------------------------------------------------ recurrences
class Rec:
    """A recurrence over `streams` sequences of n rows, and its oracle."""

    def __init__(self, rig, type_, kind, heads, dim, vdim, n, streams=2, groups=0, seed=0, gates=None):
        self.rig, self.ctx, self.type, self.kind, self.heads, self.dim, self.vdim, self.n, self.streams = rig, rig["ctx"], type_, kind, heads, dim, vdim, n, streams
        rng, self.keys = np.random.default_rng(seed), groups or heads
        kd, inner = self.keys * dim, heads * vdim
        (self.q, self.qu), (self.k, self.ku), (self.v, self.vu) = (quantise(rng.standard_normal((streams, n, w)), type_) for w in (kd, kd, inner))
        width = {REC_FORGET: heads * dim, REC_MLSTM: 2 * heads, REC_SSD: heads}[kind]
        self.gate = (rng.standard_normal((streams, n, width)) * 2 + {REC_FORGET: 1, REC_MLSTM: 0, REC_SSD: -2}[kind]).astype(np.float32)
        if gates is not None:
            self.gate = gates(self.gate).astype(np.float32)
        self.lower = rng.uniform(0, 0.8, heads * dim).astype(np.float32)
        self.a_log, self.skip = rng.uniform(-1, 1.5, heads).astype(np.float32), rng.standard_normal(heads).astype(np.float32)
        self.cap, self.ring = 6.0, 4
        copies, vp = (vdim + 31) // 32, (vdim + 3) // 4 * 4
        self.state = self.ctx.zeroed(streams * self.ring * heads * dim * vp * 4)
        self.norm, self.top = self.ctx.zeroed(streams * self.ring * heads * copies * dim * 4), self.ctx.zeroed(streams * self.ring * heads * copies * 8)
        self.consts = [f32(self.ctx, a) for a in (self.lower, self.a_log, self.skip)]

    def want(self, s):
        H, D, E, n, per = self.heads, self.dim, self.vdim, self.n, self.heads // self.keys
        q, k = (np.repeat(a[s].reshape(n, self.keys, D), per, axis=1) for a in (self.q, self.k))
        v, g = self.v[s].reshape(n, H, E), self.gate[s].astype(np.float64)
        if self.kind == REC_FORGET:
            f = self.lower + (1.0 - self.lower.astype(np.float64)) * to.sigmoid(g)
            f = f.reshape(n, H, D)
            return to.decayed_outer_products(to.silu(q), 1.0 - f, v, f).reshape(n, -1)
        if self.kind == REC_SSD:
            dt = to.softplus(g)
            decay = np.exp(-np.exp(self.a_log.astype(np.float64)) * dt)
            return (to.decayed_outer_products(q, k * dt[..., None], v, np.broadcast_to(decay[..., None], k.shape)) + self.skip[:, None] * v).reshape(n, -1)
        q = q * D ** -0.5
        i, f = self.cap * np.tanh(g[:, :H] / self.cap), to.log_sigmoid(self.cap * np.tanh(g[:, H:] / self.cap))
        S, norm, top, o = np.zeros((H, D, E)), np.zeros((H, D)), np.zeros(H), np.zeros((n, H, E))
        for t in range(n):
            new = np.maximum(f[t] + top, i[t])
            keep, write, top = np.exp(f[t] + top - new), np.exp(i[t] - new), new
            S, norm = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :], keep[:, None] * norm + write[:, None] * k[t]
            o[t] = np.einsum("hde,hd->he", S, q[t]) / (np.maximum(np.abs((norm * q[t]).sum(1)), np.exp(-top)) + 1e-6)[:, None]
        return o.reshape(n, -1)

    def run(self, at, m, chunked, streams=None):
        """Rows at .. at + m of the streams listed."""
        from turbospark_b200.capi import Recurrence
        ctx, streams = self.ctx, list(range(self.streams)) if streams is None else streams
        cut = lambda a: np.ascontiguousarray(a[streams, at:at + m].reshape(len(streams) * m, -1))

        def wide(a):
            a = cut(a)
            p = np.zeros((a.shape[0], (a.shape[1] + 15) // 16 * 16), dtype=a.dtype)
            p[:, :a.shape[1]] = a
            return ctx.to_device(p), p.shape[1]
        (q, qs), (k, ks), (v, vs), (g, gs) = wide(self.qu), wide(self.ku), wide(self.vu), wide(self.gate)
        n, inner = len(streams) * m, self.heads * self.vdim
        os_ = (inner + 15) // 16 * 16
        out = ctx.zeroed(n * os_ * 4)
        scratch = ctx.recurrence_scratch(self.kind, self.heads, self.dim, self.vdim, n, m) if chunked else ctx.zeroed(16)
        r = Recurrence(kind=self.kind, heads=self.heads, dim=self.dim, vdim=self.vdim, heads_per_key=self.heads // self.keys, cap=self.cap,
                       q_scale=self.dim ** -0.5 if self.kind == REC_MLSTM else 0.0, q=q.ptr, k=k.ptr, v=v.ptr, q_stride=qs, k_stride=ks, v_stride=vs, gate=g.ptr, gate_stride=gs,
                       lower=self.consts[0].ptr, a_log=self.consts[1].ptr, skip=self.consts[2].ptr, out=out.ptr, out_stride=os_, state=self.state.ptr, norm=self.norm.ptr,
                       top=self.top.ptr, ring=self.ring, n_streams=self.streams, scratch=scratch.ptr)
        ctx.recurrence_rows(self.type, r, ctx.to_device(descs(self.rig["tsb"], [(s, at, m) for s in streams])), n, m, chunked=chunked)
        return fetch(out, F32, (len(streams), m, os_))[:, :, :inner]


SIZES = [(REC_FORGET, 3, 24, 40, 0), (REC_FORGET, 2, 128, 128, 0), (REC_FORGET, 1, 64, 72, 0), (REC_MLSTM, 3, 24, 40, 0), (REC_MLSTM, 2, 64, 128, 0), (REC_MLSTM, 1, 128, 64, 0),
         (REC_MLSTM, 1, 200, 96, 0), (REC_SSD, 6, 24, 16, 2), (REC_SSD, 4, 128, 64, 1), (REC_SSD, 2, 256, 72, 2), (REC_SSD, 3, 16, 8, 3)]


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("kind,heads,dim,vdim,groups", SIZES + [(REC_FORGET, 1, 300, 33, 0), (REC_MLSTM, 2, 7, 5, 0), (REC_SSD, 2, 1000, 30, 1)])
def test_recurrences_row_by_row(rig, type_, kind, heads, dim, vdim, groups):
    r = Rec(rig, type_, kind, heads, dim, vdim, 40, groups=groups)
    got = [r.run(at, m, False) for at, m in portions_of(40, [1, 1, 2, 3, 9, 1, 17, 6])]
    for s in range(2):
        close(np.concatenate(got, axis=1)[s], r.want(s), 2e-5)  # f32 throughout, also with bfloat16 inputs


@pytest.mark.parametrize("kind,heads,dim,vdim,groups", SIZES)
def test_recurrences_chunk_by_chunk(rig, kind, heads, dim, vdim, groups):
    """Portions on both sides of whole chunks, single rows in between, the state carried over."""
    n = 330
    r = Rec(rig, BF16, kind, heads, dim, vdim, n, groups=groups, seed=1)
    got = [r.run(at, m, m >= 32) for at, m in portions_of(n, [64, 1, 32, 65, 2, 127, 39])]
    for s in range(2):
        close(np.concatenate(got, axis=1)[s], r.want(s), 3e-4)


@pytest.mark.parametrize("kind,dim,vdim", [(REC_FORGET, 64, 64), (REC_MLSTM, 64, 64), (REC_SSD, 64, 64)])
def test_streams_apart_equal_streams_together(rig, kind, dim, vdim):
    a, b = (Rec(rig, BF16, kind, 2, dim, vdim, 140, streams=3, seed=2) for _ in range(2))
    together = np.concatenate([a.run(0, 100, True), a.run(100, 40, True)], axis=1)
    for s in (2, 0, 1):
        alone = np.concatenate([b.run(0, 100, True, [s]), b.run(100, 40, True, [s])], axis=1)[0]
        assert np.array_equal(alone, together[s])


@pytest.mark.parametrize("dim,strength", [(128, 4.0), (64, 30.0), (40, 1000.0), (128, 0.0)])
def test_forget_gates_that_close(rig, dim, strength):
    """Gates that let little or nothing through: chunks whose decays leave the range of exponents, rows that forget everything."""
    def gates(g):
        rng = np.random.default_rng(9)
        g = g - strength
        g[:, 70:75] = 40.0        # rows that keep everything
        g[:, 20] = -200.0         # a row that forgets everything
        g[:, :, ::7] += strength  # channels that do not close
        g[:, rng.integers(0, 150, 5)] = -60.0
        return g
    r = Rec(rig, BF16, REC_FORGET, 2, dim, 64, 150, seed=3, gates=gates)
    r.lower[:] = np.where(np.arange(r.lower.size) % 3, 0.0, r.lower)
    r.consts[0] = f32(r.ctx, r.lower)
    got = [r.run(at, m, True) for at, m in portions_of(150, [64, 86])]
    for s in range(2):
        close(np.concatenate(got, axis=1)[s], r.want(s), 3e-4)


@pytest.mark.parametrize("kind", [REC_FORGET, REC_MLSTM, REC_SSD])
@pytest.mark.parametrize("chunked", [False, True])
def test_a_far_row_is_remembered(rig, kind, chunked):
    """Gates that keep nearly everything, and one strong row far back: its share is still there."""
    keep = {REC_FORGET: 12.0, REC_MLSTM: 8.0, REC_SSD: -9.0}[kind]
    r = Rec(rig, BF16, kind, 1, 64, 64, 400, streams=1, seed=4, gates=lambda g: np.full_like(g, keep))
    if kind == REC_MLSTM:
        r.gate[..., 0] = -2.0
    if kind != REC_FORGET:
        r.k[0, 3] *= 16.0
    r.v[0, 3] *= 16.0
    for x in ("k", "v"):
        v, u = quantise(getattr(r, x), BF16)
        setattr(r, x, v), setattr(r, x + "u", u)
    got = np.concatenate([r.run(at, m, chunked) for at, m in portions_of(400, [37, 200, 163])], axis=1)[0]
    want = r.want(0)
    close(got, want, 3e-4 if chunked else 2e-5)
    r.v[0, 3] = 0.0
    assert np.abs(r.want(0)[-1] - want[-1]).max() > 0.05 * np.abs(want[-1]).max()


# ------------------------------------------------------------------ experts
ROUTING = [(12, 2, 4, 3), (6, 3, 2, 1), (1, 1, 1, 1), (64, 8, 8, 4), (130, 5, 13, 4), (300, 7, 300, 50), (5, 5, 1, 1), (128, 6, 1, 1), (1024, 8, 32, 4)]


@pytest.mark.parametrize("experts,top,groups,keep", ROUTING)
@pytest.mark.parametrize("rows", [1, 7, 40, 333])
def test_choice_of_experts_and_lists(rig, experts, top, groups, keep, rows):
    from turbospark_b200.capi import ExpertLists
    ctx, rng = rig["ctx"], np.random.default_rng(experts * 1000 + rows)
    z, corr = rng.standard_normal((rows, experts)).astype(np.float32) * 2, rng.uniform(-2.5, 0.6, experts).astype(np.float32)  # choices below zero too
    if rows > 1:
        z[1] = 0.25  # ties of the scores
    lists = ExpertLists(ctx, rows, top, experts)
    ctx.route_experts(f32(ctx, z), f32(ctx, corr), experts, top, groups, keep, rows, 8, lists)
    b = lists.buffers
    ids = b["ids"].download(np.int32, rows * top).reshape(rows, top)
    s = to.sigmoid(z.astype(np.float64))
    want = to.choose_experts(s.astype(np.float32), corr, groups, keep, top)
    assert np.array_equal(ids, want)
    weight = b["weight"].download(np.float32, rows * top).reshape(rows, top)
    assert np.allclose(weight, np.take_along_axis(s, want, 1), rtol=1e-6)
    first, slot, token = b["first"].download(np.int32, experts + 1), b["slot_of"].download(np.int32, rows * top), b["token_of"].download(np.int32, rows * top)
    counts = np.bincount(ids.ravel(), minlength=experts)
    assert np.array_equal(first, np.concatenate([[0], np.cumsum(counts)]))
    order = np.argsort(ids.ravel(), kind="stable")  # an expert's slots in row order
    assert np.array_equal(np.argsort(order), slot) and np.array_equal(token, order // top)
    n = int(b["n_chunks"].download(np.int32, 1)[0])
    chunks = b["chunks"].download(np.int32, 3 * n).reshape(n, 3)
    assert np.array_equal(chunks, [(e, first[e] + i, min(8, counts[e] - i)) for e in range(experts) for i in range(0, counts[e], 8)])
    lists.free()


@pytest.mark.parametrize("type_,tensor", [(F32, False), (BF16, False), (BF16, True)])
@pytest.mark.parametrize("experts,top,d,ff,rows", [(6, 3, 96, 40, 5), (10, 2, 200, 136, 33), (4, 2, 512, 256, 150), (3, 1, 64, 64, 700), (40, 4, 128, 24, 60)])
def test_grouped_products(rig, type_, tensor, experts, top, d, ff, rows):
    """Gate-up pairs by token and by slot, then the down product; experts without tokens, experts with several tiles of them."""
    from turbospark_b200.capi import ExpertLists
    ctx, rng = rig["ctx"], np.random.default_rng(d)
    skew = np.where(np.arange(experts) % 3 == 1, -9.0, 0.0).astype(np.float32)  # some experts meet few tokens or none
    z = (rng.standard_normal((rows, experts)) + np.linspace(2, 0, experts)).astype(np.float32)
    lists = ExpertLists(ctx, rows, top, experts)
    few = 64 if type_ == F32 else 8 if rows <= 8 else 16
    ctx.route_experts(f32(ctx, z), f32(ctx, skew), experts, top, 1, 1, rows, few, lists)
    slots = rows * top
    first, token = lists.buffers["first"].download(np.int32, experts + 1), lists.buffers["token_of"].download(np.int32, slots)
    dp, fp, dr = (d + 63) // 64 * 64, (ff + 63) // 64 * 64, (d + 127) // 128 * 128
    x, xu = quantise(rng.standard_normal((rows, d)), type_)
    (gw, gu), (uw, uu), (ow, ou) = (quantise(rng.standard_normal((experts, r, c)) / c ** 0.5, type_) for r, c in ((ff, d), (ff, d), (d, ff)))
    wi, wo = np.zeros((experts, 2 * fp, dp), dtype=gu.dtype), np.zeros((experts, dr, fp), dtype=gu.dtype)
    for i in range(ff):
        wi[:, i // 8 * 16 + i % 8, :d], wi[:, i // 8 * 16 + 8 + i % 8, :d] = gu[:, i], uu[:, i]
    wo[:, :d, :ff] = ou
    alloc = max(slots, rows) + 256
    xp = np.zeros((alloc, dp), dtype=xu.dtype)
    xp[:len(token) if tensor else rows, :d] = xu[token] if tensor else xu
    a, y = ctx.zeroed(alloc * fp * 4), ctx.zeroed(alloc * d * 4)
    ctx.plain_gemm_experts(type_, ctx.to_device(wi), experts, 2 * fp, dp, ctx.to_device(xp), dp, alloc, not tensor, lists, slots, few, tensor, True, a, fp, fp)
    ctx.plain_gemm_experts(type_, ctx.to_device(wo), experts, dr, fp, a, fp, alloc, False, lists, slots, few, tensor, False, y, d, d)
    want_a, want_y = np.zeros((slots, ff)), np.zeros((slots, d))
    got_a, got_y = fetch(a, type_, (alloc, fp))[:slots, :ff], fetch(y, type_, (alloc, d))[:slots]
    for e in range(experts):
        t = slice(first[e], first[e + 1])
        want_a[t] = to.silu(x[token[t]] @ gw[e].T) * (x[token[t]] @ uw[e].T)
        want_y[t] = got_a[t] @ ow[e].T
    close(got_a, want_a, RELATIVE[type_])
    close(got_y, want_y, RELATIVE[type_])
    lists.free()


# ------------------------------------------------------------------ chunked attention with a linear bias
@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("heads,kv_heads,dim,chunk", [(6, 3, 32, 37), (8, 1, 64, 64), (8, 2, 128, 100), (20, 1, 96, 130), (4, 4, 64, 1), (2, 1, 192, 90), (12, 2, 64, 10 ** 6)])
@pytest.mark.parametrize("groups", [[(0, 250, 1), (1, 0, 1), (2, 127, 1)], [(0, 190, 7), (2, 60, 7)], [(1, 0, 300), (0, 64, 2), (2, 33, 129)]])
def test_chunked_attention(rig, type_, heads, kv_heads, dim, chunk, groups):
    """Decoded tokens, verify passes and prompt portions, one key at each end of the visible run standing out."""
    rng, ctx = np.random.default_rng(heads * dim), rig["ctx"]
    cache = Cache(rig, type_, kv_heads, dim, dim, [300, 300, 300], rng)
    n = sum(g[2] for g in groups)
    q = rng.standard_normal((n, heads, dim))
    r = 0
    for s, b, m in groups:  # queries that look for the first visible key, or for the one before it
        for i in range(m):
            p = b + i
            target = p - p % chunk - (i % 2)
            if target >= 0:
                q[r + i, i % heads] += 3.0 * cache.rows[s][target, i % heads // (heads // kv_heads), :dim]
        r += m
    sink, slopes, gate = rng.uniform(-1, 3, heads), to.alibi_slopes(heads), rng.standard_normal((n, heads, dim))
    qp, stride = padded(q.reshape(n, -1), type_)
    gp, gs = padded(gate.reshape(n, -1), type_)
    out = ctx.zeroed(n * heads * dim * 4)
    ctx.plain_attention(cache.kv, 1, ctx.to_device(qp), stride, out, heads * dim, ctx.to_device(descs(rig["tsb"], groups)), [g[2] for g in groups], heads, dim ** -0.5,
                        max(b + m for _, b, m in groups), rig["attn"], sink=f32(ctx, sink), slopes=f32(ctx, slopes), value_gate=ctx.to_device(gp), value_gate_stride=gs,
                        chunk=chunk, out_scale=0.8)
    got = fetch(out, type_, (n, heads, dim))
    qv, gv = quantise(q, type_)[0], quantise(gate, type_)[0]
    r = 0
    for s, b, m in groups:
        rows = cache.rows[s][:b + m]
        whole = np.zeros((b + m, heads, dim))
        whole[b:] = qv[r:r + m]
        want = to.chunked_attention(whole, rows[..., :dim], rows[..., dim:], dim ** -0.5, chunk, slopes.astype(np.float32).astype(np.float64), sink.astype(np.float32))[b:]
        want = want * to.sigmoid(gv[r:r + m]) * 0.8
        err = np.abs(got[r:r + m] - want).max()
        assert err < (2e-5 if type_ == F32 else 3e-2), (s, err)
        r += m
    cache.kv.close()
