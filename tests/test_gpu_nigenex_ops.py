"""The mechanisms of the plain-weight decoders as operators, against the plain float64 oracle."""
import numpy as np
import pytest

from oracle import nigenex_oracle as no
from turbospark_b200.plain import BF16, F32, GELU_TANH, SILU, bf16_bits, bf16_to_f32

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def rig():
    import turbospark_b200 as tsb
    ctx = tsb.Ctx(0)
    yield dict(tsb=tsb, ctx=ctx, ws=ctx.plain_gemm_workspace(), attn=ctx.window_attention_scratch())
    ctx.close()


def quantise(x, type_):
    """The values a tensor of this type holds, and what is uploaded for them."""
    x = np.asarray(x, dtype=np.float32)
    if type_ == F32:
        return x.astype(np.float64), x
    b = bf16_bits(x).reshape(x.shape)
    return bf16_to_f32(b).reshape(x.shape).astype(np.float64), b


def fetch(buf, type_, shape):
    n = int(np.prod(shape))
    return buf.download(np.float32, n).reshape(shape) if type_ == F32 else bf16_to_f32(buf.download(np.uint16, n)).reshape(shape)


def descs(tsb, groups):
    """groups: (stream, base, rows) -> device row descriptors of chains."""
    return tsb.row_descs([(s, b, j, b + j, 0) for s, b, n in groups for j in range(n)])


# ------------------------------------------------------------------ matmul
@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("tokens", [1, 7, 8, 9, 16, 17, 32, 33, 64, 65, 127, 129, 257, 600])
def test_matmul_at_every_token_count_around_the_kernels_edges(rig, type_, tokens):
    ctx, rng = rig["ctx"], np.random.default_rng(tokens)
    rows, cols, valid = 384, 320, 333
    wv, wu = quantise(rng.standard_normal((rows, cols)), type_)
    x_rows = max(32, tokens) + 3
    xv, xu = quantise(rng.standard_normal((x_rows, cols)), type_)
    y0 = rng.standard_normal((tokens, valid)).astype(np.float32)
    w, x = ctx.to_device(wu), ctx.to_device(xu)
    want = xv[:tokens] @ wv[:valid].T
    tol = 2e-5 * np.sqrt(cols)
    y = ctx.to_device(np.full((tokens + 1, valid), 77.0, dtype=np.float32))
    ctx.plain_gemm(type_, w, rows, cols, x, x_rows, tokens, y, valid, valid, rig["ws"])
    got = y.download(np.float32, (tokens + 1) * valid).reshape(tokens + 1, valid)
    assert np.abs(got[:tokens] - want).max() < tol and np.all(got[tokens] == 77.0)
    y.upload(y0)
    ctx.plain_gemm(type_, w, rows, cols, x, x_rows, tokens, y, valid, valid, rig["ws"], add=True)
    assert np.abs(y.download(np.float32, tokens * valid).reshape(tokens, valid) - (y0 + want)).max() < tol
    ctx.plain_gemm(type_, w, rows, cols, x, x_rows, tokens, y, valid, valid, rig["ws"], cap=9.0)
    assert np.abs(y.download(np.float32, tokens * valid).reshape(tokens, valid) - no.soft_cap(want, 9.0)).max() < tol


@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("tokens", [1, 20, 40, 100, 300])
def test_long_products_are_cut_along_the_columns_and_repeat(rig, type_, tokens):
    """Few row tiles and many columns: the tensor-memory kernel cuts the columns into runs; the result is the same again."""
    ctx, rng = rig["ctx"], np.random.default_rng(5)
    rows, cols = 128, 4160
    wv, wu = quantise(rng.standard_normal((rows, cols)) / np.sqrt(cols), type_)
    xv, xu = quantise(rng.standard_normal((320, cols)), type_)
    w, x, y = ctx.to_device(wu), ctx.to_device(xu), ctx.alloc(tokens * rows * 4)
    outs = []
    for _ in range(3):
        ctx.plain_gemm(type_, w, rows, cols, x, 320, tokens, y, rows, rows, rig["ws"])
        outs.append(y.download(np.float32, tokens * rows).reshape(tokens, rows))
    assert np.abs(outs[0] - xv[:tokens] @ wv.T).max() < 5e-5
    assert np.array_equal(outs[0], outs[1]) and np.array_equal(outs[0], outs[2])


@pytest.mark.parametrize("act", [GELU_TANH, SILU])
@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("tokens,pairs", [(1, 64), (13, 100), (50, 192), (200, 8)])
def test_gate_up_pairs(rig, type_, act, tokens, pairs):
    ctx, rng = rig["ctx"], np.random.default_rng(pairs)
    cols, padded = 192, (pairs + 63) // 64 * 64
    gv, _ = quantise(rng.standard_normal((padded, cols)) * 0.2, type_)
    uv, _ = quantise(rng.standard_normal((padded, cols)) * 0.1, type_)
    packed = np.stack([gv.reshape(-1, 8, cols), uv.reshape(-1, 8, cols)], axis=1).reshape(2 * padded, cols)
    _, wu = quantise(packed, type_)
    xv, xu = quantise(rng.standard_normal((max(32, tokens), cols)), type_)
    a = ctx.zeroed(tokens * padded * 4)
    ctx.plain_gemm_pairs(type_, ctx.to_device(wu), 2 * padded, cols, ctx.to_device(xu), max(32, tokens), tokens, a, padded, pairs, act, rig["ws"])
    got = fetch(a, type_, (tokens, padded))
    g, u = xv[:tokens] @ gv.T, xv[:tokens] @ uv.T
    want = (no.gelu_tanh(g) if act == GELU_TANH else g / (1 + np.exp(-g))) * u
    tol = 2e-5 if type_ == F32 else 2 ** -8 * np.abs(want[:, :pairs]).max()
    assert np.abs(got[:, :pairs] - want[:, :pairs]).max() < tol and np.all(got[:, pairs:] == 0)


# ------------------------------------------------------------------ norm and token shift
@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("d", [64, 200, 1030])
def test_norm_and_shift_carry_the_row_before_through_portions_and_reused_streams(rig, type_, d):
    tsb, ctx, rng = rig["tsb"], rig["ctx"], np.random.default_rng(d)
    ring, streams, eps, gain = 8, 3, 1e-2, 1.3
    mu = rng.uniform(0, 1, d).astype(np.float32)
    state = ctx.zeroed(streams * ring * d * 4)
    state.upload(np.full(streams * ring * d, 1e6, dtype=np.float32))  # what an earlier request left behind
    gd, md = ctx.to_device(np.array([gain], dtype=np.float32)), ctx.to_device(mu)
    seqs = {s: rng.standard_normal((30, d)).astype(np.float32) for s in range(streams)}
    at = {s: 0 for s in range(streams)}

    def run(groups, x, use_mu=True):
        n = x.shape[0]
        mix, h = ctx.zeroed(n * d * 4), ctx.zeroed(n * d * 4)
        ctx.norm_shift_rows(type_, ctx.to_device(x), d, gd, eps, md if use_mu else None, ctx.to_device(descs(tsb, groups)), n, state, streams, ring,
                            mix, h, d)
        return fetch(mix, type_, (n, d)), fetch(h, type_, (n, d))

    tol = 3e-6 if type_ == F32 else 2 ** -7
    for sizes in [{0: 3, 2: 1}, {2: 2, 1: 7, 0: 1}, {0: 1}, {0: 1, 1: 1, 2: 1}, {2: 7, 0: 5}, {1: 2}]:
        groups = [(s, at[s], n) for s, n in sizes.items()]
        mix, h = run(groups, np.concatenate([seqs[s][b:b + n] for s, b, n in groups]))
        r = 0
        for s, b, n in groups:
            full = no.rms_norm_scalar(seqs[s].astype(np.float64), gain, eps)
            assert np.abs(h[r:r + n] - full[b:b + n]).max() < tol * 4
            assert np.abs(mix[r:r + n] - no.token_shift(full, mu.astype(np.float64))[b:b + n]).max() < tol * 4
            r += n
            at[s] += n
    # a new request in a used stream starts from zeros; a rewound one from the row that is still kept
    full = no.rms_norm_scalar(seqs[0].astype(np.float64), gain, eps)
    mix, _ = run([(1, 0, 2)], seqs[0][:2])
    assert np.abs(mix - no.token_shift(full, mu.astype(np.float64))[:2]).max() < tol * 4
    mix, _ = run([(0, at[0] - 3, 2)], seqs[0][at[0] - 3:at[0] - 1])
    assert np.abs(mix - no.token_shift(full, mu.astype(np.float64))[at[0] - 3:at[0] - 1]).max() < tol * 4
    mix, h = run([(0, 5, 1)], seqs[0][5:6], use_mu=False)
    assert np.array_equal(mix, h)


# ------------------------------------------------------------------ attention
class Cache:
    """Streams of random keys in a paged key cache whose pages are handed out in a shuffled order."""

    def __init__(self, rig, type_, kv_heads, dim, lengths, rng, page=64, boost=None):
        from turbospark_b200.capi import KeyCache
        pages = [(n + page - 1) // page for n in lengths]
        self.kv = KeyCache(rig["ctx"], type_, 2, kv_heads, dim, page, sum(pages) + 3, len(lengths), max(pages))
        self.keys = []
        for step in range(max(pages)):  # streams grow in turn, so their pages interleave
            for s in rng.permutation(len(lengths)):
                if step < pages[s]:
                    self.kv.reserve(int(s), min((step + 1) * page, lengths[s]))
        for s, n in enumerate(lengths):
            k = rng.standard_normal((n, kv_heads, dim))
            if boost:
                boost(s, k)
            v, u = quantise(k, type_)
            self.keys.append(v)
            self.kv.write_rows(s, 1, 0, u.reshape(n, -1))


def attend(rig, type_, cache, groups, q, heads, scale, cap, r1, r2, gate, window, q_stride=None):
    tsb, ctx = rig["tsb"], rig["ctx"]
    n, _, dim = q.shape
    _, qu = quantise(q, type_)
    up = lambda a: None if a is None else ctx.to_device(np.asarray(a, dtype=np.float32))
    stride = (heads * dim + 15) // 16 * 16
    padded = np.zeros((n, stride), dtype=qu.dtype)
    padded[:, :heads * dim] = qu.reshape(n, -1)
    out = ctx.zeroed(n * stride * 4)
    ctx.window_attention(cache.kv, 1, ctx.to_device(padded), stride, out, stride, ctx.to_device(descs(tsb, groups)),
                         [g[2] for g in groups], heads, scale, cap, up(r1), up(r2), up(gate), window, max(b + m for _, b, m in groups), rig["attn"])
    return fetch(out, type_, (n, stride))[:, :heads * dim].reshape(n, heads, dim)


def expect(cache, groups, q, scale, cap, r1, r2, gate, window, type_):
    qv, _ = quantise(q, type_)
    out, r = [], 0
    for s, b, n in groups:
        k = cache.keys[s][:b + n]
        H = q.shape[1]
        c = cap if cap > 0 else 1e9
        z = np.zeros(H)
        out.append(no.attention(qv[r:r + n], k, k, scale, c, z if r1 is None else r1, z if r2 is None else r2, window or 10 ** 9, first_query=b))
        r += n
    o = np.concatenate(out)
    return o if gate is None else no.head_gate(o, np.asarray(gate, dtype=np.float64))


@pytest.mark.parametrize("type_,heads,kv_heads,dim", [(BF16, 8, 2, 64), (BF16, 6, 2, 32), (BF16, 5, 1, 96), (BF16, 4, 4, 128), (BF16, 4, 1, 192),
                                                      (BF16, 2, 1, 256), (BF16, 24, 1, 64), (BF16, 80, 1, 32), (F32, 8, 2, 64), (F32, 3, 3, 20),
                                                      (F32, 4, 1, 260)])
@pytest.mark.parametrize("window", [0, 1, 2, 63, 64, 65, 130])
def test_attention_over_unequal_portions(rig, type_, heads, kv_heads, dim, window):
    rng = np.random.default_rng(heads * 1000 + dim + window)
    lengths = [1, 5, 64, 65, 200, 333]
    cache = Cache(rig, type_, kv_heads, dim, lengths, rng)
    scale, cap = 1.5 / np.sqrt(dim), 4.0
    r1, r2 = rng.uniform(0, 1.5, heads), rng.uniform(0.05, 0.6, heads)
    tol = 2e-5 if type_ == F32 else 2e-2
    for sizes in [[1, 1, 1, 1, 1, 1], [1, 2, 33, 1, 60, 150], [None, 5, 64, None, None, 333], [None, None, 3, 3, 3, 3]]:
        groups = [(s, lengths[s] - n, n) for s, n in enumerate(sizes) if n]
        rows = sum(n for _, _, n in groups)
        q = rng.standard_normal((rows, heads, dim))
        gate = rng.standard_normal((rows, heads)) * 2
        got = attend(rig, type_, cache, groups, q, heads, scale, cap, r1, r2, gate, window)
        want = expect(cache, groups, q, scale, cap, r1.astype(np.float32), r2.astype(np.float32), gate.astype(np.float32), window, type_)
        assert np.abs(got - want).max() < tol, (sizes, np.abs(got - want).max())
    cache.kv.close()


@pytest.mark.parametrize("scale,cap", [(0.01, 50.0), (0.2, 50.0), (2.0, 50.0), (0.5, 1.0), (30.0, 20.0), (-0.4, 6.0)])
@pytest.mark.parametrize("dim", [64, 128])
@pytest.mark.parametrize("rows", [1, 10, 100])
def test_scores_far_inside_and_far_beyond_the_cap(rig, rows, dim, scale, cap):
    """The many-query kernel has a series for small scores and the exponential form for the rest: both, and tiles that mix."""
    rng = np.random.default_rng(rows)
    cache = Cache(rig, BF16, 2, dim, [300], rng)
    q = rng.standard_normal((rows, 8, dim)) / np.sqrt(dim / 64)
    q[:, 3] *= 0.01
    r = np.full(8, 0.2, dtype=np.float32)
    groups = [(0, 300 - rows, rows)]
    got = attend(rig, BF16, cache, groups, q, 8, scale, cap, r, r, None, 200)
    assert np.abs(got - expect(cache, groups, q, scale, cap, r, r, None, 200, BF16)).max() < 2.5e-2
    cache.kv.close()


@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("rows", [1, 2, 40])
def test_cap_bias_and_gate_are_optional_one_by_one(rig, type_, rows):
    rng = np.random.default_rng(rows)
    cache = Cache(rig, type_, 2, 64, [150, 90], rng)
    groups = [(0, 150 - rows, rows), (1, 90 - rows, rows)]
    q = rng.standard_normal((2 * rows, 4, 64))
    r1, r2 = np.array([0.1, 1, 2, 0.02]), np.array([0.5, 0.1, 0.3, 0.2])
    gate = rng.standard_normal((2 * rows, 4))
    seen = []
    for cap, bias, g in [(0.0, False, None), (1.5, False, None), (0.0, True, None), (0.0, False, gate), (1.5, True, gate)]:
        a = (0.2, cap, r1 if bias else None, r2 if bias else None, g, 100)
        got = attend(rig, type_, cache, groups, q, 4, *a)
        assert np.abs(got - expect(cache, groups, q, *a, type_)).max() < (2e-5 if type_ == F32 else 2e-2)
        seen.append(got)
    assert all(np.abs(a - b).max() > 0.02 for i, a in enumerate(seen) for b in seen[i + 1:])
    cache.kv.close()


@pytest.mark.parametrize("type_", [BF16, F32])
@pytest.mark.parametrize("window", [64, 97, 300])
@pytest.mark.parametrize("portion", [1, 2, 31, 200])
def test_a_key_that_stands_out_counts_just_inside_the_window_and_not_outside(rig, type_, window, portion):
    """One key carries nearly all of the weight of the queries that see it: at the window's edge, at page borders, far back
    and at the query itself, for decoded rows and for every row of a portion."""
    rng = np.random.default_rng(window)
    heads, kv_heads, dim, n = 4, 2, 64, 500
    spike = np.zeros(dim)
    spike[3] = 30.0
    for at in [0, 1, 63, 64, 127, 191, 192, 250, 255, 256, 257, 319, 448]:
        def boost(s, k, at=at):
            k *= 0.3
            k[at] = spike
        cache = Cache(rig, type_, kv_heads, dim, [n], rng, boost=boost)
        q = rng.standard_normal((portion, heads, dim)) * 0.1
        q[:, :, 3] = 4.0
        for last in sorted({min(n - 1, max(portion - 1, at + d)) for d in (0, 1, window - 1, window, window + 1, window + portion // 2)}):
            groups = [(0, last + 1 - portion, portion)]
            r1, r2 = np.full(heads, 0.3), np.full(heads, 0.2)
            got = attend(rig, type_, cache, groups, q, heads, 0.5, 40.0, r1, r2, None, window)
            want = expect(cache, groups, q, 0.5, 40.0, r1.astype(np.float32), r2.astype(np.float32), None, window, type_)
            assert np.abs(got - want).max() < (1e-3 if type_ == F32 else 0.15), (at, last)
            for i in range(portion):
                dist = last + 1 - portion + i - at
                assert (got[i, :, 3].min() > 20) == (0 <= dist < window), (at, last, i)
        cache.kv.close()


def test_long_contexts_are_cut_into_runs_and_repeat(rig):
    rng = np.random.default_rng(9)
    cache = Cache(rig, BF16, 2, 128, [5000, 3], rng)
    for window, rows in [(0, 1), (4096, 1), (1000, 12), (0, 100), (4500, 5)]:
        groups = [(0, 5000 - rows, rows), (1, 2, 1)]
        q = rng.standard_normal((rows + 1, 8, 128))
        a = (0.3, 10.0, np.full(8, 0.2, dtype=np.float32), np.full(8, 0.1, dtype=np.float32), None, window)
        got = attend(rig, BF16, cache, groups, q, 8, *a)
        assert np.abs(got - expect(cache, groups, q, *a, BF16)).max() < 2e-2
        assert np.array_equal(got, attend(rig, BF16, cache, groups, q, 8, *a))
    cache.kv.close()


def test_operators_refuse_what_they_do_not_cover(rig):
    tsb, ctx = rig["tsb"], rig["ctx"]
    from turbospark_b200.capi import KeyCache, KvCache
    with pytest.raises(tsb.TsbError):
        KeyCache(ctx, BF16, 1, 1, 40, 64, 4, 1, 4)  # heads are stored padded
    b = ctx.zeroed(1 << 16)
    with pytest.raises(tsb.TsbError):
        ctx.plain_gemm(BF16, b, 100, 64, b, 32, 1, b, 64, 64, rig["ws"])
    with pytest.raises(tsb.TsbError):
        ctx.plain_gemm(BF16, b, 128, 64, b, 8, 1, b, 64, 64, rig["ws"])
    kv = KvCache(ctx, 1, 1, 64, 64, 4, 1, 4)
    with pytest.raises(tsb.TsbError):
        ctx.window_attention(kv, 0, b, 64, b, 64, b, [1], 1, 1.0, 0.0, None, None, None, 0, 1, rig["attn"])
    keys = KeyCache(ctx, BF16, 1, 1, 64, 64, 4, 1, 4)
    with pytest.raises(tsb.TsbError):
        ctx.attn_decode_rows(keys, 0, b, 64, b, b, 1, 1, 4, 1.0, 1, b)
    with pytest.raises(tsb.TsbError):
        ctx.window_attention(keys, 0, b, 64, b, 64, b, [1], 200, 1.0, 0.0, None, None, None, 0, 1, rig["attn"])
    with pytest.raises(tsb.TsbError, match="32-byte"):
        ctx.window_attention(keys, 0, b, 72, b, 64, b, [1], 1, 1.0, 0.0, None, None, None, 0, 1, rig["attn"])
    kv.close(), keys.close()
