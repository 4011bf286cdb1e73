// Attention over a plain paged cache (attention_window.cuh): this unit has the kernels for caches whose values are their keys, the
// f32 kernel and the merge; attention_kv.cu has the kernels for caches with values of their own, attention_prefix.cu those with a prefix.
//
// bfloat16: one kernel template <D, MT, SL> on mma.sync m16n8k16.  A CTA owns one (query tile, key head, run of key tiles):
// MT m-tiles of 16 queries - the tile's rows x the heads that share the key head - and walks 64-token key tiles that
// cp.async brings into a three-stage ring.  The one tile in shared memory serves both products: K rows as the B operand
// of S = Q K^T (ldmatrix) and as the B operand of O += P K (ldmatrix.trans), so a key byte is read once.  SL warps share an
// m-tile, each taking 64 / SL tokens of every tile, and meet at the end.
//   few queries (short portions): MT = 1 or 4, SL = 4 or 2; many queries whose geometry the tcgen05 kernel (attention_window_tc.cu) does
//   not take: MT = 8, SL = 1
// Up to eight queries per key head (decoded tokens), and 17 to 32 (verify passes) with heads of up to 128 columns, go to
// window_attn_few_kernel: keys on the M side.
// A context that does not fill the device with CTAs is cut into runs of key tiles: with up to eight queries the last CTA of a
// tile to finish - decided by a ticket, nobody waits - adds the runs in order, with more a merge launch does.
// Only the key tiles inside the window of some query of the tile are visited; key tiles start at multiples of 64 positions
// whatever the cut of the prompt, so a row meets its keys in the same grouping in every schedule.
//
// Score arithmetic in f32, base 2: v = cap log2(e) tanh(s scale / cap) - r1 log2(1 + r2 d); tanh by a polynomial where every
// score of the warp's tile is well inside the cap.
//
// f32: one warp per (row, query head), lanes over keys for the scores and over columns for the sum; the reference-precision
// mode, plain fused multiply-adds and the library's exp, tanh and log.
#include <algorithm>

#include "attention_window_mma.cuh"

namespace {

// ------------------------------------------------------------------ merge of cut tiles
// One CTA per row and eight query heads, a warp per head: the runs' weights sit in the lanes, the sums go over the runs in order.
__global__ void __launch_bounds__(256)
    window_attn_merge_kernel(const __grid_constant__ WindowAttn a, const AttnTile* __restrict__ tiles, int tiles_per_group, int rows_per_seq,
                             int rows_per_tile, int n_splits, int slots, const float* __restrict__ part_o, const float2* __restrict__ part_ml) {
    const int tile = blockIdx.x, r = blockIdx.y;
    int row_first, n_rows;
    if (tiles) {
        row_first = tiles[tile].row_first, n_rows = tiles[tile].n_rows;
    } else {
        const int in_group = (tile % tiles_per_group) * rows_per_tile;
        row_first = (tile / tiles_per_group) * rows_per_seq + in_group;
        n_rows = min(rows_per_tile, rows_per_seq - in_group);
    }
    pdl_wait();
    pdl_launch_dependents();
    if (r >= n_rows) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int D = a.value_dim > 0 ? a.value_dim : a.keys.head_dim, grp = a.n_q_heads / a.keys.kv_heads, R = WATTN_LARGE_Q / grp;
    const int head = blockIdx.z * 8 + warp;
    if (head < a.n_q_heads) {
        const int slot = (r / R) * WATTN_LARGE_Q + (r % R) * grp + head % grp;
        const int64_t first = ((int64_t)tile * a.keys.kv_heads + head / grp) * n_splits * slots + slot;
        float2 v[WATTN_MAX_SPLITS / 32];
        float m = -INFINITY, l = 0.f;
#pragma unroll
        for (int i = 0; i < WATTN_MAX_SPLITS / 32; i++) {
            const int k = i * 32 + lane;
            v[i] = k < n_splits ? part_ml[first + (int64_t)k * slots] : make_float2(-INFINITY, 0.f);
            m = fmaxf(m, v[i].x);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        const float mu = m == -INFINITY ? 0.f : m;
#pragma unroll
        for (int i = 0; i < WATTN_MAX_SPLITS / 32; i++) v[i].x = ex2(v[i].x - mu), l = fmaf(v[i].y, v[i].x, l);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
        const float f = head_factor(a, row_first + r, head, m, l);
        __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (int64_t)(row_first + r) * a.out_stride + (int64_t)head * D;
        for (int c0 = 0; c0 < D; c0 += 128) {
            const int c = c0 + lane * 4;
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
            for (int k = 0; k < n_splits; k++) {
                const float w = __shfl_sync(0xffffffffu, k < 32 ? v[0].x : v[1].x, k & 31);
                if (c < D) {
                    const float4 x = *reinterpret_cast<const float4*>(part_o + (first + (int64_t)k * slots) * D + c);
                    acc.x = fmaf(x.x, w, acc.x), acc.y = fmaf(x.y, w, acc.y), acc.z = fmaf(x.z, w, acc.z), acc.w = fmaf(x.w, w, acc.w);
                }
            }
            if (c < D && a.turn) turn_back(a, row_first + r, c, acc.x, acc.y), turn_back(a, row_first + r, c + 2, acc.z, acc.w);
            if (c < D && a.value_gate) value_gates(a, row_first + r, head, c, acc);
            if (c < D) *reinterpret_cast<uint2*>(out + c) = make_uint2(pack_bf16(acc.x * f, acc.y * f), pack_bf16(acc.z * f, acc.w * f));
        }
    }
}

// ------------------------------------------------------------------ f32
constexpr int F32_WARPS = 4;
constexpr int F32_MAX_DIM = 512;   // columns of a value
constexpr int F32_MAX_KEY = 1024;  // columns of a key
__global__ void __launch_bounds__(F32_WARPS * 32) window_attn_f32_kernel(const __grid_constant__ WindowAttn a, int rows, uint32_t* __restrict__ err) {
    __shared__ float qs[F32_WARPS][F32_MAX_KEY];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t item = (int64_t)blockIdx.x * F32_WARPS + warp;
    pdl_wait();
    pdl_launch_dependents();
    if (item >= (int64_t)rows * a.n_q_heads) return;
    const int row = (int)(item / a.n_q_heads), head = (int)(item % a.n_q_heads);
    const int D = a.keys.head_dim, DV = a.value_dim > 0 ? a.value_dim : D, kvh = head / (a.n_q_heads / a.keys.kv_heads);
    const tsb_row_desc rd = a.rows[row];
    const int pos = rd.base + rd.slot;
    const float* q = reinterpret_cast<const float*>(a.q) + (int64_t)row * a.q_stride + (int64_t)head * D;
    for (int i = lane; i < D; i += 32) qs[warp][i] = q[i];
    __syncwarp();
    const int lo = first_visible(a, pos);
    const float slope = a.slopes ? a.slopes[head] : 0.f;
    const float r1 = a.r1 ? a.r1[head] : 0.f, r2 = a.r1 ? a.r2[head] : 0.f;
    // a sink is a score without a key or a value: it opens the sum
    float m = a.sink ? a.sink[head] : -INFINITY, l = a.sink ? 1.f : 0.f, acc[F32_MAX_DIM / 32];
#pragma unroll
    for (int i = 0; i < F32_MAX_DIM / 32; i++) acc[i] = 0.f;
    // first what is seen of the prefix, then the window
    const int n_pre = a.window > 0 && (a.keep > 0 || a.pool > 0) ? prefix_len(a, pos) : 0, pre_end = (n_pre + 31) & ~31;
    for (int i0 = 0; i0 < pre_end + pos + 1 - (lo & ~31); i0 += 32) {
        const bool pre = i0 < pre_end;
        const int j0 = pre ? i0 : i0 - pre_end + (lo & ~31), j = j0 + lane;
        const KeyView& rows_of = pre && a.pool > 0 ? a.pooled : a.keys;
        const bool seen = pre ? j < n_pre : j >= lo && j <= pos;
        const float* k = seen ? key_row<float>(rows_of, rd.seq, j) : nullptr;
        if (seen && !k) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        float s = -INFINITY;
        if (k) {
            k += (int64_t)kvh * a.keys.head_step;
            float4 dot = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int i = 0; i < D; i += 4) {
                const float4 v = *reinterpret_cast<const float4*>(k + i);
                dot.x = fmaf(v.x, qs[warp][i], dot.x), dot.y = fmaf(v.y, qs[warp][i + 1], dot.y);
                dot.z = fmaf(v.z, qs[warp][i + 2], dot.z), dot.w = fmaf(v.w, qs[warp][i + 3], dot.w);
            }
            s = ((dot.x + dot.y) + (dot.z + dot.w)) * a.scale;
            if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
            if (a.r1) s -= r1 * logf(1.f + r2 * (float)(pos - j));
            if (a.slopes) s -= slope * (float)(pos - j);
        }
        float mx = s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_new = fmaxf(m, mx);
        if (m_new == -INFINITY) continue;
        const float alpha = expf(m - m_new), p = expf(s - m_new);
        m = m_new;
        float ps = p;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
        l = fmaf(l, alpha, ps);
#pragma unroll
        for (int i = 0; i < F32_MAX_DIM / 32; i++) acc[i] *= alpha;
        for (int t = 0; t < 32; t++) {
            const float pt = __shfl_sync(0xffffffffu, p, t);
            if (pt == 0.f) continue;  // the same for every lane
            const float* kt = key_row<float>(rows_of, rd.seq, j0 + t);
            if (!kt) continue;
            kt += (int64_t)kvh * a.keys.head_step + a.keys.value_off;
#pragma unroll
            for (int i = 0; i < F32_MAX_DIM / 32; i++)
                if (i * 32 + lane < DV) acc[i] = fmaf(pt, kt[i * 32 + lane], acc[i]);
        }
    }
    const float f = (l > 0.f ? a.out_scale / l : 0.f) * (a.gate ? sigmoid(a.gate[(int64_t)row * a.n_q_heads + head]) : 1.f);
    float* out = reinterpret_cast<float*>(a.out) + (int64_t)row * a.out_stride + (int64_t)head * DV;
    const float* vg = a.value_gate ? reinterpret_cast<const float*>(a.value_gate) + (int64_t)row * a.value_gate_stride + (int64_t)head * DV : nullptr;
#pragma unroll
    for (int i = 0; i < F32_MAX_DIM / 32; i++)
        if (i * 32 < DV) {
            float v = acc[i];
            if (a.turn) {  // the columns of a pair sit in neighbouring lanes
                float u = __shfl_xor_sync(0xffffffffu, v, 1);
                if (lane & 1) turn_back(a, row, i * 32 + lane - 1, u, v);
                else turn_back(a, row, i * 32 + lane, v, u);
            }
            if (i * 32 + lane < DV) out[i * 32 + lane] = v * f * (vg ? sigmoid(vg[i * 32 + lane]) : 1.f);
        }
}

}  // namespace

cudaError_t launch_window_attn_merge(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int splits, int slots, const WattnScratch& sc) {
    return tsb_launch(ctx, window_attn_merge_kernel, dim3((unsigned)l.n_tiles, (unsigned)l.rows_per_tile, (unsigned)((a.n_q_heads + 7) / 8)), dim3(256), 0, st, true, a, l.tiles,
                      l.tiles_per_group, l.rows_per_seq, l.rows_per_tile, splits, slots, (const float*)sc.o, (const float2*)sc.ml);
}

size_t wattn_scratch_bytes(const tsb_ctx* ctx) {
    return WATTN_TICKETS * sizeof(uint32_t) + wattn_part_queries(ctx) * (sizeof(float2) + 256 * sizeof(float));
}

int wattn_rows_per_tile(int head_dim, int group, bool biased) {
    const int per = WATTN_LARGE_Q / group > 0 ? WATTN_LARGE_Q / group : 1;
    return wattn_tc_supported(head_dim, group, biased) ? 2 * per : per;
}

int wattn_pad_dim(int head_dim, bool f32) {
    if (head_dim <= 0) return 0;
    if (f32) return head_dim <= F32_MAX_DIM ? (head_dim + 3) / 4 * 4 : 0;
    for (int d : {32, 64, 96, 128, 192, 256})
        if (head_dim <= d) return d;
    return 0;
}

bool wattn_supported(int head_dim, int group, bool f32) { return wattn_pad_dim(head_dim, f32) > 0 && group >= 1 && (f32 || group <= WATTN_LARGE_Q); }

cudaError_t launch_window_attn(tsb_ctx* ctx, cudaStream_t st, bool f32, const WindowAttn& a, const AttnBatch& b, void* scratch) {
    if (has_prefix(a) && (a.window <= 0 || a.keys.value_off == 0 || a.r1 || a.slopes || (a.keep > 0 && a.pool > 0))) return cudaErrorInvalidValue;
    if (f32)
        return tsb_launch(ctx, window_attn_f32_kernel, dim3((unsigned)(((int64_t)b.rows * a.n_q_heads + F32_WARPS - 1) / F32_WARPS)), dim3(F32_WARPS * 32),
                          0, st, true, a, b.rows, ctx->dev_error);
    const int grp = a.n_q_heads / a.keys.kv_heads, rpt = wattn_rows_per_tile(a.keys.head_dim, grp, a.r1 != nullptr);
    const bool kv = a.keys.value_off > 0, pre = has_prefix(a);
    auto large = [&](const WattnLaunch& l) {
        if (wattn_tc_supported(a.keys.head_dim, grp, a.r1 != nullptr)) return (pre ? launch_prefix_attn_tc : kv ? launch_kv_attn_tc : launch_window_attn_tc)(ctx, st, a, l, scratch);
        if (pre) return launch_prefix_attn_large(ctx, st, a, l, scratch);
        return kv ? launch_kv_attn_large(ctx, st, a, l, scratch) : launch_large<8, 1, false>(ctx, st, a, l, scratch);
    };
    auto small = [&](const WattnLaunch& l, int queries) {
        if (pre) return launch_prefix_attn_small(ctx, st, a, l, queries, scratch);
        return kv ? launch_kv_attn_small(ctx, st, a, l, queries, scratch) : launch_small<false>(ctx, st, a, l, queries, scratch);
    };
    if (b.rows_per_seq > 0) {
        const int groups = b.rows / b.rows_per_seq, queries = b.rows_per_seq * grp;
        if (queries <= WATTN_SMALL_Q) return small(WattnLaunch{nullptr, groups, 1, b.rows_per_seq, b.rows_per_seq, b.max_len}, queries);
        const int tpg = (b.rows_per_seq + rpt - 1) / rpt;
        return large(WattnLaunch{nullptr, groups * tpg, tpg, b.rows_per_seq, rpt, b.max_len});
    }
    cudaError_t e = cudaSuccess;
    if (b.n_large > 0) e = large(WattnLaunch{b.large, b.n_large, 1, 0, rpt, b.max_len});
    if (e == cudaSuccess && b.n_small > 0) e = small(WattnLaunch{b.small, b.n_small, 1, 0, WATTN_SMALL_Q / grp, b.max_len}, b.small_queries);
    return e;
}
