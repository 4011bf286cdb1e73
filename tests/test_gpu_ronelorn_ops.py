"""Windows with a prefix, turning values, norms followed by rotations, block means, element-wise recurrences, products with an activation or scaled
sums as operators, against the plain float64 oracle."""
import numpy as np
import pytest

from oracle import ronelorn_oracle as ro
from tests.test_gpu_gimozen_ops import f32, padded, upload
from tests.test_gpu_nigenex_ops import descs, fetch, quantise
from tests.test_gpu_tarivik_ops import close, portions_of
from turbospark_b200.plain import BF16, F32, GELU_TANH, RELU2, SILU

pytestmark = pytest.mark.gpu
RELATIVE = {F32: 3e-6, BF16: 9e-3}


@pytest.fixture(scope="module")
def rig():
    import turbospark_b200 as tsb
    ctx = tsb.Ctx(0)
    yield dict(tsb=tsb, ctx=ctx, attn=ctx.window_attention_scratch(), gemm=ctx.plain_gemm_workspace())
    ctx.close()


def values_of(rows, type_):
    return rows.astype(np.float64) if type_ == F32 else (rows.astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def side_by_side(x, dims):
    """Halves of the first `dims` columns -> pairs next to each other."""
    half = dims // 2
    order = [i // 2 + (i % 2) * half for i in range(dims)] + list(range(dims, x.shape[-1]))
    return x[..., order]


def table(positions, freq):
    a = np.asarray(positions, dtype=np.float64)[:, None] * freq
    return np.stack([np.cos(a), np.sin(a)], axis=-1).astype(np.float32)


class Blocks:
    """Streams of random rows of heads * [key, value] and the means of their blocks, pages handed out in a shuffled order."""

    def __init__(self, rig, type_, heads, key_dim, value_dim, lengths, pool, rng, page=64):
        from turbospark_b200.capi import PlainCache
        self.pages = [(n + page - 1) // page for n in lengths]
        self.kv = PlainCache(rig["ctx"], type_, 2, heads, key_dim, value_dim, page, sum(self.pages) + 3, len(lengths), max(self.pages), pool=pool)
        for step in range(max(self.pages)):  # streams grow in turn, so their pages interleave
            for s in rng.permutation(len(lengths)):
                if step < self.pages[s]:
                    self.kv.reserve(int(s), min((step + 1) * page, lengths[s]))
        self.rows = []
        for s, n in enumerate(lengths):
            v, u = quantise(rng.standard_normal((n, heads, key_dim + value_dim)), type_)
            self.rows.append(v)
            self.kv.write_rows(s, 1, 0, u.reshape(n, -1))


# ------------------------------------------------------------------ block means
@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("pool,page", [(16, 64), (5, 64), (1, 64), (70, 64), (200, 16), (3, 16), (64, 64), (24, 128)])
def test_block_means(rig, type_, pool, page):
    """Every block of portions that start and end anywhere, whatever pages the rows and the blocks are in."""
    ctx, rng, heads, dim = rig["ctx"], np.random.default_rng(pool), 3, 32
    lengths = [211, 64, 400]
    c = Blocks(rig, type_, heads, dim, dim, lengths, pool, rng, page)
    for sizes in ([100, 1, 1, 1, 45, 2, 300],):
        at = 0
        for m in sizes:
            groups = [(s, at, min(m, n - at)) for s, n in enumerate(lengths) if at < n]
            ctx.block_mean_rows(c.kv, 1, ctx.to_device(descs(rig["tsb"], groups)), sum(g[2] for g in groups))
            at += m
    for s, n in enumerate(lengths):
        if n // pool == 0:
            continue
        got = values_of(c.kv.read_blocks(s, 1, 0, n // pool), type_)
        close(got, ro.block_means(c.rows[s], pool).reshape(n // pool, -1), RELATIVE[type_])
    c.kv.close()


# ------------------------------------------------------------------ attention
GEOMETRY = [(6, 3, 32), (8, 2, 64), (8, 1, 128), (4, 4, 96), (20, 1, 64), (2, 1, 192), (3, 3, 256), (32, 4, 128)]
BATCHES = [[(0, 350, 1), (1, 0, 1), (2, 157, 1)], [(0, 190, 7), (2, 60, 7)], [(1, 0, 300), (0, 64, 2), (2, 33, 129)], [(0, 399, 1), (2, 100, 290)], [(0, 0, 400)]]


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("heads,kv_heads,dim", GEOMETRY)
@pytest.mark.parametrize("groups", BATCHES)
@pytest.mark.parametrize("window,prefix", [(37, ("keep", 5)), (64, ("keep", 64)), (100, ("keep", 130)), (1, ("keep", 1)), (300, ("keep", 1000)), (37, ("pool", 5)), (64, ("pool", 16)),
                                           (1, ("pool", 1)), (130, ("pool", 70)), (90, ("pool", 3)), (50, ("pool", 300))])
def test_window_with_a_prefix(rig, type_, heads, kv_heads, dim, groups, window, prefix):
    """Decoded tokens, verify passes and prompt portions; queries look for one key just inside or just outside what they see: the ends of the window, of the kept
    tokens and of the blocks."""
    kind, size = prefix
    rng, ctx = np.random.default_rng(heads * dim + window), rig["ctx"]
    pool = size if kind == "pool" else 0
    lengths = [400, 300, 400]
    c = Blocks(rig, type_, kv_heads, dim, dim, lengths, pool, rng)
    if pool:
        for s, n in enumerate(lengths):
            ctx.block_mean_rows(c.kv, 1, ctx.to_device(descs(rig["tsb"], [(s, 0, n)])), n)
    means = [values_of(c.kv.read_blocks(s, 1, 0, n // pool), type_).reshape(-1, kv_heads, 2 * dim) if pool and n >= pool else np.zeros((0, kv_heads, 2 * dim))
             for s, n in enumerate(lengths)]
    n = sum(g[2] for g in groups)
    q = rng.standard_normal((n, heads, dim)) * 0.5
    r = 0
    for s, b, m in groups:
        for i in range(m):
            p, h = b + i, i % heads
            g = h // (heads // kv_heads)
            before = max(0, p - window + 1)
            targets = [c.rows[s][t, g, :dim] for t in (before, before - 1) if 0 <= t <= p]
            if pool:
                targets += [means[s][t, g, :dim] * pool ** 0.5 for t in (before // pool - 1, before // pool) if 0 <= t < len(means[s])]
            else:
                targets += [c.rows[s][t, g, :dim] for t in (size - 1, size) if t <= p]
            q[r + i, h] += 3.0 * targets[(i // heads) % len(targets)]
        r += m
    cap, sink = (6.0, None) if pool else (0.0, np.zeros(heads))
    half = dim // 4  # the last columns of a head do not turn
    turn = table(np.concatenate([b + np.arange(m) for _, b, m in groups]), ro.frequencies(50.0, 2 * half))
    qp, stride = padded(q.reshape(n, -1), type_)
    out = ctx.zeroed(n * heads * dim * 4)
    ctx.plain_attention(c.kv, 1, ctx.to_device(qp), stride, out, heads * dim, ctx.to_device(descs(rig["tsb"], groups)), [g[2] for g in groups], heads, dim ** -0.5,
                        max(b + m for _, b, m in groups), rig["attn"], cap=cap, window=window, sink=f32(ctx, sink), keep=0 if pool else size, blocks=bool(pool),
                        turn=f32(ctx, turn), turn_half=half)
    got = fetch(out, type_, (n, heads, dim))
    qv = quantise(q, type_)[0]
    r = 0
    for s, b, m in groups:
        rows, pos = c.rows[s][:b + m], np.arange(b, b + m)
        if pool:
            blocks = means[s][:(b + m) // pool]
            both = np.concatenate([blocks, rows])
            seen = np.concatenate([ro.block_mask(b + m, window, pool)[:, :len(blocks)], ro.window_mask(b + m, window)], axis=1)[b:]
        else:
            both, seen = rows, ro.kept_mask(b + m, window, size)[b:]
        want = ro.grouped_attention(qv[r:r + m], both[..., :dim], both[..., dim:], seen, dim ** -0.5, cap=cap or None, one_more=not pool)
        cs, sn = turn[r:r + m, None, :, 0].astype(np.float64), turn[r:r + m, None, :, 1].astype(np.float64)
        u, v = want[..., 0:2 * half:2].copy(), want[..., 1:2 * half:2].copy()
        want[..., 0:2 * half:2], want[..., 1:2 * half:2] = u * cs + v * sn, v * cs - u * sn
        err = np.abs(got[r:r + m] - want).max()
        assert err < (3e-5 if type_ == F32 else 3e-2), (s, err)
        r += m
    c.kv.close()


def test_a_prefix_that_no_kernel_has_is_refused(rig):
    ctx, rng = rig["ctx"], np.random.default_rng(0)
    c = Blocks(rig, BF16, 1, 64, 64, [64], 0, rng)
    q = ctx.zeroed(64 * 2)
    args = (c.kv, 1, q, 64, q, 64, ctx.to_device(descs(rig["tsb"], [(0, 10, 1)])), [1], 1, 0.1, 64, rig["attn"])
    for extras in (dict(keep=3), dict(keep=3, window=5, slopes=q), dict(window=5, blocks=True), dict(window=5, keep=-1)):
        with pytest.raises(rig["tsb"].TsbError):
            ctx.plain_attention(*args, **extras)
    with pytest.raises(rig["tsb"].TsbError):
        c.kv.read_blocks(0, 1, 0, 1)
    with pytest.raises(rig["tsb"].TsbError):
        ctx.block_mean_rows(c.kv, 1, ctx.to_device(descs(rig["tsb"], [(0, 10, 1)])), 1)
    c.kv.close()


# ------------------------------------------------------------------ norms and rotations
@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("projection", [False, True])
@pytest.mark.parametrize("nq,nk,width,vwidth,rot", [(6, 3, 40, 24, 20), (32, 8, 128, 128, 128), (5, 1, 25, 30, 10), (4, 2, 160, 64, 6), (3, 3, 64, 128, 0), (8, 2, 18, 6, 2)])
def test_norms_rotations_and_turned_values(rig, type_, projection, nq, nk, width, vwidth, rot):
    from turbospark_b200.capi import PlainCache
    ctx, rng, n, eps = rig["ctx"], np.random.default_rng(width), 11, 1e-3
    pad = (max(width, vwidth) + 31) // 32 * 32
    kv = PlainCache(ctx, type_, 1, nk, pad, pad, 16, 4, 2, 2)
    kv.reserve(0, 20), kv.reserve(1, 20)
    nv, wide = (0, nq * width, ) if projection else (nk, width)
    raw = rng.standard_normal((2 * n, (nq + nk) * width + nv * vwidth)).astype(np.float32)
    wq, wk = rng.uniform(0.5, 1.5, nq * width if projection else width).astype(np.float32), rng.uniform(0.5, 1.5, nk * width if projection else width).astype(np.float32)
    pos = np.concatenate([5 + np.arange(n), np.arange(n)])
    rt, tt = table(pos, ro.frequencies(77.0, rot, 1.7)), table(pos, ro.frequencies(77.0, vwidth))
    q = ctx.to_device(np.full(2 * n * nq * pad * 4, 0x7f, dtype=np.uint8))
    ctx.turned_norm_rows(kv, 0, f32(ctx, raw), raw.shape[1], nq, nk, width, f32(ctx, wq), f32(ctx, wk), eps, ctx.to_device(descs(rig["tsb"], [(1, 5, n), (0, 0, n)])), 2 * n, q,
                         nq * pad, rot=f32(ctx, rt) if rot else None, rot_half=rot // 2, n_v=nv, v_width=vwidth, turn=f32(ctx, tt) if nv else None, turn_half=vwidth // 2,
                         projection=projection)

    def turned(x, t):  # pairs side by side
        y, half = x.copy(), t.shape[1]
        c, s = t[:, None, :, 0].astype(np.float64), t[:, None, :, 1].astype(np.float64)
        u, v = x[..., 0:2 * half:2], x[..., 1:2 * half:2]
        y[..., 0:2 * half:2], y[..., 1:2 * half:2] = u * c - v * s, v * c + u * s
        return y

    def normed(x, w, heads):
        x = x.astype(np.float64)
        x = ro.rms(x, eps) * w if projection else ro.rms(x.reshape(2 * n, heads, width), eps) * w
        return turned(x.reshape(2 * n, heads, width), rt)
    got = fetch(q, type_, (2 * n, nq, pad))
    close(got[..., :width].reshape(2 * n, -1), normed(raw[:, :nq * width], wq, nq).reshape(2 * n, -1), RELATIVE[type_])
    assert not got[..., width:].any()
    keys = normed(raw[:, nq * width:(nq + nk) * width], wk, nk)
    for s, base, first in ((1, 5, 0), (0, 0, n)):
        rows = values_of(kv.read_rows(s, 0, base, n), type_).reshape(n, nk, 2, pad)
        close(rows[:, :, 0, :width].reshape(n, -1), keys[first:first + n].reshape(n, -1), RELATIVE[type_])
        if nv:
            want = turned(raw[first:first + n, (nq + nk) * width:].astype(np.float64).reshape(n, nk, vwidth), tt[first:first + n])
            close(rows[:, :, 1, :vwidth].reshape(n, -1), want.reshape(n, -1), RELATIVE[type_])
    kv.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("d", [200, 4096, 75, 5120])
def test_pre_norm_leaves_the_stream(rig, type_, d):
    ctx, rng, n, eps = rig["ctx"], np.random.default_rng(d), 9, 1e-4
    x, w = (rng.standard_normal((n, d)) * rng.uniform(0.1, 9, (n, 1))).astype(np.float32), rng.uniform(0.5, 1.5, d).astype(np.float32)
    stride = (d + 15) // 16 * 16
    xd, out = f32(ctx, x), ctx.zeroed(n * stride * 4)
    ctx.pre_norm_rows(type_, xd, d, f32(ctx, w), eps, n, out, stride)
    close(fetch(out, type_, (n, stride))[:, :d], ro.shifted_rms_norm(x.astype(np.float64), w - 1.0, eps), RELATIVE[type_])
    assert np.array_equal(fetch(xd, F32, (n, d)), x)


# ------------------------------------------------------------------ products
@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("tokens", [1, 9, 33, 130, 300])
@pytest.mark.parametrize("cols", [64, 320, 1024])
def test_products_with_an_activation_and_scaled_sums(rig, type_, tokens, cols):
    ctx, rng, rows, valid = rig["ctx"], np.random.default_rng(tokens + cols), 256, 200
    alloc = max(32, (tokens + 31) // 32 * 32)
    w, wu = quantise(rng.standard_normal((rows, cols)) / cols ** 0.5, type_)
    x, xu = quantise(rng.standard_normal((alloc, cols)), type_)
    wd, xd = ctx.to_device(wu), ctx.to_device(xu)
    z = x[:tokens] @ w[:valid].T
    for act, f in ((RELU2, ro.squared_relu), (SILU, ro.silu), (GELU_TANH, lambda v: 0.5 * v * (1 + np.tanh((2 / np.pi) ** 0.5 * (v + 0.044715 * v ** 3))))):
        y = ctx.zeroed(tokens * valid * 4)
        ctx.plain_gemm_act(type_, wd, rows, cols, xd, alloc, tokens, y, valid, valid, act, rig["gemm"])
        close(fetch(y, type_, (tokens, valid)), f(z), RELATIVE[type_])
    y0 = rng.standard_normal((tokens, valid)).astype(np.float32)
    y = f32(ctx, y0)
    ctx.plain_gemm_add(type_, wd, rows, cols, xd, alloc, tokens, y, valid, valid, 0.5, 0.3, rig["gemm"])
    close(fetch(y, F32, (tokens, valid)), 0.5 * y0 + 0.3 * z, 3e-6)


# ------------------------------------------------------------------ element-wise recurrence
@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("width,sizes", [(136, [1] * 9 + [2, 7, 40, 31, 33]), (57, [500]), (2048, [128, 1, 129, 31]), (5000, [64, 3]), (8, [300, 5000, 1, 1]), (4100, [1, 32])])
def test_gated_scan(rig, type_, chunked, width, sizes):
    """Three streams in the portions given, the state carried over in a ring that wraps; channels that keep next to everything and channels that keep nothing."""
    ctx, rng, n, streams = rig["ctx"], np.random.default_rng(width), sum(sizes), 3
    z = (rng.standard_normal((streams, n, width)) * 2 + np.linspace(-9, 6, width)).astype(np.float32)
    u = (rng.standard_normal((streams, n, width)) * 2).astype(np.float32)
    g, gu = quantise(rng.standard_normal((streams, n, width)) * 2, type_)
    s = np.stack([ro.gated_scan(ro.sigmoid(z[i].astype(np.float64)), ro.positive(u[i].astype(np.float64))) for i in range(streams)])
    want = s * ro.silu(g)
    ring, pitch, stride = 4, (width + 3) // 4 * 4, (width + 15) // 16 * 16
    state = ctx.to_device(rng.standard_normal(streams * ring * pitch).astype(np.float32))  # what an earlier request left
    order = [2, 0, 1]
    for at, m in portions_of(n, sizes):
        gate = np.concatenate([z[order, at:at + m], u[order, at:at + m]], axis=-1).reshape(streams * m, 2 * width)
        gp = np.zeros((streams * m, stride), dtype=gu.dtype)
        gp[:, :width] = gu[order, at:at + m].reshape(-1, width)
        out = ctx.zeroed(streams * m * stride * 4)
        ctx.gated_scan_rows(type_, f32(ctx, gate), 2 * width, ctx.to_device(gp), stride, width, state, streams, ring, ctx.to_device(descs(rig["tsb"], [(i, at, m) for i in order])),
                            streams * m, m, out, stride, chunked=chunked, sums=ctx.zeroed(streams * (m // 128 + 1) * width * 8))
        got, w = fetch(out, type_, (streams * m, stride))[:, :width], want[order, at:at + m].reshape(-1, width)
        assert (np.abs(got - w) <= (3e-5 if type_ == F32 else 5e-3) * np.abs(w) + 3e-5).all()
        kept = fetch(state, F32, (streams, ring, pitch))
        for p in range(max(at, at + m - ring), at + m):  # every position of the ring
            assert np.allclose(kept[:, p % ring, :width], s[:, p], rtol=3e-5, atol=1e-6)
