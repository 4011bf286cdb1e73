"""Attention over keys and values and over latent rows, products per head and norms as operators, against the plain float64 oracle."""
import numpy as np
import pytest

from oracle import gimozen_oracle as go
from tests.test_gpu_nigenex_ops import descs, fetch, quantise
from turbospark_b200.plain import BF16, F32

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def rig():
    import turbospark_b200 as tsb
    ctx = tsb.Ctx(0)
    yield dict(tsb=tsb, ctx=ctx, ws=ctx.plain_gemm_workspace(), attn=ctx.window_attention_scratch())
    ctx.close()


class Cache:
    """Streams of random rows of heads * [key, value] in a cache whose pages are handed out in a shuffled order.  value_dim 0: latent
    rows of key_dim numbers of which the first `latent` are the value."""

    def __init__(self, rig, type_, heads, key_dim, value_dim, lengths, rng, page=64, boost=None, used=None):
        from turbospark_b200.capi import PlainCache
        pages = [(n + page - 1) // page for n in lengths]
        self.kv = PlainCache(rig["ctx"], type_, 2, heads, key_dim, value_dim, page, sum(pages) + 3, len(lengths), max(pages))
        self.rows = []
        for step in range(max(pages)):  # streams grow in turn, so their pages interleave
            for s in rng.permutation(len(lengths)):
                if step < pages[s]:
                    self.kv.reserve(int(s), min((step + 1) * page, lengths[s]))
        for s, n in enumerate(lengths):
            k = rng.standard_normal((n, heads, key_dim + value_dim))
            if used:
                k[:, :, used:key_dim] = 0.0  # padding columns
            if boost:
                boost(s, k)
            v, u = quantise(k, type_)
            self.rows.append(v)
            self.kv.write_rows(s, 1, 0, u.reshape(n, -1))


def upload(ctx, x, type_):
    return ctx.to_device(quantise(x, type_)[1])


def padded(x, type_):
    """[rows, n] with a row stride that is a multiple of 16 -> uploaded values, stride."""
    _, u = quantise(x, type_)
    stride = (u.shape[1] + 15) // 16 * 16
    p = np.zeros((u.shape[0], stride), dtype=u.dtype)
    p[:, :u.shape[1]] = u
    return p, stride


def f32(ctx, a):
    return None if a is None else ctx.to_device(np.asarray(a, dtype=np.float32))


def value_attention(rig, type_, cache, groups, q, value_dim, scale, sink=None, gate=None, window=0):
    ctx, (n, heads, dim) = rig["ctx"], q.shape
    qp, stride = padded(q.reshape(n, -1), type_)
    ostride = (heads * value_dim + 15) // 16 * 16
    out = ctx.zeroed(n * ostride * 4)
    extra = {}
    if gate is not None:
        gp, gs = padded(gate.reshape(n, -1), type_)
        extra = dict(value_gate=ctx.to_device(gp), value_gate_stride=gs)
    ctx.plain_attention(cache.kv, 1, ctx.to_device(qp), stride, out, ostride, ctx.to_device(descs(rig["tsb"], groups)), [g[2] for g in groups], heads, scale,
                        max(b + m for _, b, m in groups), rig["attn"], sink=f32(ctx, sink), window=window, **extra)
    return fetch(out, type_, (n, ostride))[:, :heads * value_dim].reshape(n, heads, value_dim)


def latent_attention(rig, type_, cache, groups, q, value_dim, scale, sink):
    ctx, (n, heads, dim) = rig["ctx"], q.shape
    qp, stride = padded(q.reshape(n, -1), type_)
    ostride = heads * value_dim
    out = ctx.zeroed(n * ostride * 4)
    ctx.latent_attention(cache.kv, 1, ctx.to_device(qp), stride, out, ostride, ctx.to_device(descs(rig["tsb"], groups)), [g[2] for g in groups], heads,
                         value_dim, scale, f32(ctx, sink), max(b + m for _, b, m in groups), rig["attn"])
    return fetch(out, type_, (n, ostride)).reshape(n, heads, value_dim)


def expect(cache, groups, q, key_dim, values, scale, sink, type_, gate=None):
    """values: the columns of a row that are the value."""
    qv, _ = quantise(q, type_)
    out, r = [], 0
    for s, b, n in groups:
        rows = cache.rows[s][:b + n]
        out.append(go.causal_attention(qv[r:r + n], rows[:, :, :key_dim], rows[:, :, values], scale, None if sink is None else np.float32(sink).astype(np.float64),
                                       first_query=b))
        r += n
    o = np.concatenate(out)
    return o if gate is None else o * go.sigmoid(quantise(gate, type_)[0])


LENGTHS = [1, 5, 64, 65, 200, 333]
PORTIONS = [[1, 1, 1, 1, 1, 1], [1, 2, 33, 1, 60, 150], [None, 5, 64, None, None, 333], [None, None, 3, 3, 3, 3], [None, None, None, None, 129, 129]]


def groups_of(sizes):
    return [(s, LENGTHS[s] - n, n) for s, n in enumerate(sizes) if n]


@pytest.mark.parametrize("type_,heads,kv_heads,dim", [(BF16, 8, 2, 64), (BF16, 6, 2, 32), (BF16, 5, 1, 96), (BF16, 4, 4, 128), (BF16, 4, 1, 192),
                                                      (BF16, 2, 1, 256), (BF16, 24, 1, 64), (BF16, 80, 1, 32), (BF16, 32, 2, 128), (F32, 8, 2, 64),
                                                      (F32, 3, 3, 20), (F32, 4, 1, 260)])
def test_attention_over_keys_and_values(rig, type_, heads, kv_heads, dim):
    rng = np.random.default_rng(heads * 1000 + dim)
    cache = Cache(rig, type_, kv_heads, dim, dim, LENGTHS, rng)
    sink = rng.uniform(-2, 4, heads)
    for i, sizes in enumerate(PORTIONS):
        groups = groups_of(sizes)
        rows = sum(n for _, _, n in groups)
        q, gate = rng.standard_normal((rows, heads, dim)), rng.standard_normal((rows, heads, dim)) * 2
        sk, gt = (None, sink)[i % 2], (gate, None)[i % 3 == 2]
        got = value_attention(rig, type_, cache, groups, q, dim, 1.5 / np.sqrt(dim), sk, gt)
        want = expect(cache, groups, q, dim, slice(dim, None), 1.5 / np.sqrt(dim), sk, type_, gt)
        assert np.abs(got - want).max() < (2e-5 if type_ == F32 else 2e-2), (sizes, np.abs(got - want).max())
    cache.kv.close()


@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("key_dim,value_dim", [(64, 64), (64, 128), (128, 64), (128, 128), (192, 64), (192, 128)])
@pytest.mark.parametrize("page", [16, 64, 256])
def test_keys_and_values_of_different_widths(rig, type_, key_dim, value_dim, page):
    rng = np.random.default_rng(key_dim + value_dim + page)
    heads = 3
    cache = Cache(rig, type_, heads, key_dim, value_dim, LENGTHS, rng, page=page)
    sink = rng.uniform(-2, 4, heads)
    for sizes in PORTIONS[1:]:
        groups = groups_of(sizes)
        rows = sum(n for _, _, n in groups)
        q, gate = rng.standard_normal((rows, heads, key_dim)), rng.standard_normal((rows, heads, value_dim)) * 2
        a = (cache, groups, q, value_dim, 1.5 / np.sqrt(key_dim), sink, gate)
        got = value_attention(rig, type_, *a)
        want = expect(cache, groups, q, key_dim, slice(key_dim, None), 1.5 / np.sqrt(key_dim), sink, type_, gate)
        assert np.abs(got - want).max() < (2e-5 if type_ == F32 else 2e-2), (sizes, np.abs(got - want).max())
        assert np.array_equal(got, value_attention(rig, type_, *a))
    cache.kv.close()


# value columns, key columns, numbers of the row that are used
LATENTS = [(64, 64, 50), (64, 96, 90), (64, 160, 150), (128, 160, 160), (192, 192, 192), (256, 288, 288), (384, 448, 420), (512, 576, 576), (512, 640, 600)]


@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("value_dim,key_dim,used", LATENTS)
@pytest.mark.parametrize("heads", [1, 5, 32, 40])
def test_attention_over_latent_rows(rig, type_, value_dim, key_dim, used, heads):
    rng = np.random.default_rng(heads * 1000 + key_dim)
    cache = Cache(rig, type_, 1, key_dim, 0, LENGTHS, rng, used=used)
    sink = rng.uniform(-2, 4, heads)
    for sizes in PORTIONS[:4] if heads < 32 else PORTIONS[:2]:
        groups = groups_of(sizes)
        q = rng.standard_normal((sum(n for _, _, n in groups), heads, key_dim))
        a = (cache, groups, q, value_dim, 1.5 / np.sqrt(used), sink)
        got = latent_attention(rig, type_, *a)
        want = expect(cache, groups, q, key_dim, slice(0, value_dim), 1.5 / np.sqrt(used), sink, type_)
        assert np.abs(got - want).max() < (2e-5 if type_ == F32 else 2e-2), (sizes, np.abs(got - want).max())
    cache.kv.close()


@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("kind", ["values", "wide", "latent"])
@pytest.mark.parametrize("portion", [1, 2, 31, 70, 260])
def test_a_key_that_stands_out_counts_for_itself_and_everything_after_it(rig, type_, kind, portion):
    """One key carries nearly all of the weight of the queries that see it: at the borders of pages and key tiles, at the start, and at
    the query itself; the query just before it does not see it."""
    rng = np.random.default_rng(portion)
    heads, n = 4, 700
    kd, vd, kvh, values = {"values": (64, 64, 2, slice(64, None)), "wide": (192, 64, 4, slice(192, None)), "latent": (128, 0, 1, slice(0, 128))}[kind]
    for at in [0, 1, 63, 64, 127, 128, 255, 256, 511, 512, 640]:
        def boost(s, k, at=at):
            k *= 0.3
            k[at, :, 3] = 30.0
            k[at, :, kd:] = 9.0
        cache = Cache(rig, type_, kvh, kd, vd, [n], rng, boost=boost)
        q = rng.standard_normal((portion, heads, kd)) * 0.1
        q[:, :, 3] = 4.0
        for last in sorted({min(n - 1, max(portion - 1, at + d)) for d in (0, portion // 2, 300)}):
            groups = [(0, last + 1 - portion, portion)]
            if kind == "latent":
                got = latent_attention(rig, type_, cache, groups, q, 128, 0.5, np.full(heads, 1.0))
            else:
                got = value_attention(rig, type_, cache, groups, q, vd, 0.5, np.full(heads, 1.0))
            want = expect(cache, groups, q, kd, values, 0.5, np.full(heads, 1.0), type_)
            assert np.abs(got - want).max() < (1e-3 if type_ == F32 else 0.15), (at, last)
            for i in range(portion):
                big = got[i, :, 3].min() > 5
                assert big == (last + 1 - portion + i >= at), (at, last, i)
        cache.kv.close()


@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("kind", ["values", "wide", "latent"])
@pytest.mark.parametrize("rows", [1, 70])
def test_a_sink_weighs_like_a_key_without_a_value(rig, type_, kind, rows):
    """Sinks from far below every score to far above all of them, also in contexts that are cut into runs; without one the weights
    sum to one."""
    rng = np.random.default_rng(rows)
    heads, n = 4, 3000
    kd, vd, kvh = {"values": (64, 64, 2), "wide": (128, 64, 4), "latent": (96, 0, 1)}[kind]
    cache = Cache(rig, type_, kvh, kd, vd, [n, 2], rng, boost=lambda s, k: k.__setitem__((slice(None), slice(None), slice(vd and kd, None)), 1.0))
    q = rng.standard_normal((rows + 1, heads, kd)) * 0.2
    sink = np.array([-60.0, 0.0, 7.0, 80.0])
    groups = [(0, n - rows, rows), (1, 1, 1)]
    run = (lambda s: latent_attention(rig, type_, cache, groups, q, 64, 0.3, s)) if kind == "latent" else \
        (lambda s: value_attention(rig, type_, cache, groups, q, vd, 0.3, s))
    values = slice(0, 64) if kind == "latent" else slice(kd, None)
    with_sink, without = run(sink), run(None)
    assert np.abs(with_sink - expect(cache, groups, q, kd, values, 0.3, sink, type_)).max() < (1e-4 if type_ == F32 else 1e-2)
    assert np.abs(without - expect(cache, groups, q, kd, values, 0.3, None, type_)).max() < (1e-4 if type_ == F32 else 1e-2)
    assert np.abs(with_sink[:, 3]).max() < 1e-3 and np.abs(with_sink[:, 0] - without[:, 0]).max() < 1e-2
    cache.kv.close()


def test_long_contexts_are_cut_into_runs_and_repeat(rig):
    rng = np.random.default_rng(9)
    for kind, kd, vd, kvh, heads in (("values", 128, 128, 2, 8), ("wide", 192, 128, 3, 3), ("latent", 576, 0, 1, 16)):
        cache = Cache(rig, BF16, kvh, kd, vd, [5000, 3], rng)
        for rows in (1, 3, 12, 100):
            groups = [(0, 5000 - rows, rows), (1, 2, 1)]
            q, sink = rng.standard_normal((rows + 1, heads, kd)), np.full(heads, 2.0)
            if kind == "latent":
                run = lambda: latent_attention(rig, BF16, cache, groups, q, 512, 0.1, sink)
                want = expect(cache, groups, q, kd, slice(0, 512), 0.1, sink, BF16)
            else:
                run = lambda: value_attention(rig, BF16, cache, groups, q, vd, 0.2, sink)
                want = expect(cache, groups, q, kd, slice(kd, None), 0.2, sink, BF16)
            got = run()
            assert np.abs(got - want).max() < 2e-2, (kind, rows)
            assert np.array_equal(got, run())
        cache.kv.close()


# ------------------------------------------------------------------ products per head
@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("tokens", [1, 8, 9, 33, 70, 129, 300])
@pytest.mark.parametrize("heads,valid,head_rows,cols,x_step", [(3, 128, 128, 64, 64), (5, 100, 128, 128, 192), (2, 200, 256, 256, 256), (2, 20, 128, 576, 640),
                                                               (1, 384, 384, 192, 192)])
def test_products_per_head_with_and_without_gates(rig, type_, tokens, heads, valid, head_rows, cols, x_step):
    ctx, rng = rig["ctx"], np.random.default_rng(tokens + cols)
    wv, wu = quantise(rng.standard_normal((heads, head_rows, cols)) / np.sqrt(cols), type_)
    x_rows = max(32, tokens)
    xv, xu = quantise(rng.standard_normal((x_rows, heads * x_step)), type_)
    gv, gu = quantise(rng.standard_normal((tokens, heads * valid)) * 2, type_)
    y_step = head_rows + 8
    w, x, g = ctx.to_device(wu), ctx.to_device(xu), ctx.to_device(gu)
    want = np.stack([xv[:tokens, h * x_step:h * x_step + cols] @ wv[h, :valid].T for h in range(heads)], axis=1)
    for gate in (None, g):
        y = ctx.zeroed(tokens * heads * y_step * 4)
        ctx.plain_gemm_heads(type_, w, heads, head_rows, cols, x, heads * x_step, x_step, x_rows, tokens, y, heads * y_step, y_step, valid, rig["ws"], gate=gate,
                             gate_stride=heads * valid, gate_step=valid)
        got = fetch(y, type_, (tokens, heads, y_step))
        ref = want * go.sigmoid(gv.reshape(tokens, heads, valid)) if gate is not None else want
        assert np.abs(got[:, :, :valid] - ref).max() < (2e-5 if type_ == F32 else 2 ** -8 * np.abs(ref).max() + 1e-3)
        assert np.all(got[:, :, valid:] == 0)


# ------------------------------------------------------------------ norms
@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("d", [64, 200, 1030, 4100, 8192])
def test_norm_after_the_sum(rig, type_, d):
    ctx, rng = rig["ctx"], np.random.default_rng(d)
    x, w = (rng.standard_normal((7, d)) * 3).astype(np.float32), rng.uniform(0.5, 1.5, d).astype(np.float32)
    xb, out = ctx.to_device(x), ctx.zeroed(7 * (d + 8) * 4)
    ctx.post_norm_rows(type_, xb, d, ctx.to_device(w), 1e-2, 7, out, d + 8)
    want = go.rms_norm(x.astype(np.float64), w.astype(np.float64), 1e-2)
    assert np.abs(xb.download(np.float32, 7 * d).reshape(7, d) - want).max() < 2e-6 * 4
    assert np.abs(fetch(out, type_, (7, d + 8))[:, :d] - want).max() < (8e-6 if type_ == F32 else 2 ** -8 * np.abs(want).max())


@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("width,stored", [(20, 32), (64, 64), (33, 64), (128, 128), (200, 256), (256, 256)])
def test_norms_of_heads_with_query_temperature(rig, type_, width, stored):
    ctx, rng = rig["ctx"], np.random.default_rng(width)
    nq, nk, eps, coef, every = 6, 2, 1e-3, 0.7, 50
    cache = Cache(rig, type_, nk, stored, stored, [160, 70], rng)
    groups = [(0, 40, 100), (1, 60, 10)]
    n = 110
    raw = rng.standard_normal((n, nq + nk, width)).astype(np.float32)
    wq, wk = rng.uniform(0.5, 1.5, width).astype(np.float32), rng.uniform(0.5, 1.5, width).astype(np.float32)
    for temp in (every, 0):
        q = ctx.to_device(np.full(n * nq * stored, 7.0, dtype=np.float32))
        ctx.head_norm_rows(cache.kv, 1, ctx.to_device(raw), (nq + nk) * width, nq, nk, width, ctx.to_device(wq), ctx.to_device(wk), eps,
                           ctx.to_device(descs(rig["tsb"], groups)), n, q, nq * stored, temp_coef=coef, temp_every=temp)
        pos = np.concatenate([np.arange(40, 140), np.arange(60, 70)])
        want = go.rms_norm(raw[:, :nq].astype(np.float64), wq.astype(np.float64), eps)
        if temp:
            want = want * go.query_temperature(pos, coef, every)[:, None, None]
        got = fetch(q, type_, (n, nq, stored))
        tol = lambda ref: (2e-6 if type_ == F32 else 2 ** -8) * np.abs(ref).max()
        assert np.abs(got[:, :, :width] - want).max() < tol(want) and np.all(got[:, :, width:] == 0)
        keys = go.rms_norm(raw[:, nq:].astype(np.float64), wk.astype(np.float64), eps)
        r = 0
        for s, b, m in groups:
            back = cache.kv.read_rows(s, 1, b, m)
            back = (back if type_ == F32 else quantise_back(back)).reshape(m, nk, 2, stored)
            assert np.abs(back[:, :, 0, :width] - keys[r:r + m]).max() < tol(keys)
            assert np.array_equal(back[:, :, 1], cache.rows[s][b:b + m].reshape(m, nk, 2, stored)[:, :, 1])  # values stay as they are
            r += m
    cache.kv.close()


def quantise_back(bits):
    from turbospark_b200.plain import bf16_to_f32
    return bf16_to_f32(bits).reshape(bits.shape)


def test_operators_refuse_what_they_do_not_cover(rig):
    tsb, ctx = rig["tsb"], rig["ctx"]
    from turbospark_b200.capi import PlainCache
    b = ctx.zeroed(1 << 16)
    kv = PlainCache(ctx, BF16, 1, 1, 192, 128, 64, 4, 1, 4)
    with pytest.raises(tsb.TsbError):  # two query heads share a key head: not in the kernel for different widths
        ctx.plain_attention(kv, 0, b, 384, b, 256, b, [1], 2, 1.0, 1, rig["attn"])
    with pytest.raises(tsb.TsbError):
        ctx.latent_attention(kv, 0, b, 192, b, 128, b, [1], 1, 128, 1.0, None, 1, rig["attn"])
    kv.close()
    kv = PlainCache(ctx, BF16, 1, 1, 100 // 4 * 4 + 4, 0, 64, 4, 1, 4)
    with pytest.raises(tsb.TsbError):
        ctx.latent_attention(kv, 0, b, 112, b, 64, b, [1], 1, 64, 1.0, None, 1, rig["attn"])
    kv.close()
    with pytest.raises(tsb.TsbError):
        ctx.plain_gemm_heads(BF16, b, 1, 100, 64, b, 64, 64, 32, 1, b, 128, 128, 100, rig["ws"])
    with pytest.raises(tsb.TsbError):
        PlainCache(ctx, BF16, 1, 1, 36, 0, 64, 4, 1, 4)  # rows are whole 16-byte pieces
