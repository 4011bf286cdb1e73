// Attention over a plain cache for many queries (prompt portions) on the fifth-generation tensor cores, bfloat16.  Keys of DK
// and values of DV columns, multiples of 64.  KV = false: the values are the keys; KV = true: a stage holds a tile of each.
//
// A CTA owns up to 256 queries - consecutive rows of one stream x the heads of one key head, as two query tiles of 128 -
// and walks a run of key tiles of TN (64 or 128) tokens:
//   warps 0-3, 4-7  one softmax warpgroup per query tile.  A thread is a query and owns its tensor-memory lane: it reads its
//                   row of S = Q K^T (tcgen05.ld), turns it into base-2 logits (soft cap, distance bias, mask at the edges),
//                   and writes P = 2^(v - m) as bfloat16 over the scores, the A operand of the second product.  Row maxima
//                   and sums stay in the thread.  m moves only when a tile's maximum exceeds it by more than 8; only then
//                   the output accumulator is rescaled in place.
//   warp 8          fetches key tiles, a lane per box, through TMA (a 2-D map over the layer's pages, one box per page and 64
//                   columns, 128-byte swizzle).  Keys are the K-major B operand of Q K^T, values the MN-major B operand of P V:
//                   where the values are the keys the same bytes serve as both, and a tile is fetched once.
//   warp 9          (of a third warpgroup, whose other two warps only give up their registers) issues tcgen05.mma, alternating between the two query tiles: while one warpgroup works on its scores the
//                   tensor pipe has the other tile's products.
// The distance bias of a key tile takes few distinct values (rows of the tile + 127 per head): each warpgroup tabulates them
// in shared memory before its scores arrive, so the inner loop has no logarithm.
// CTAs take the tiles from the last one on: with a causal mask it has the most keys.
// A cut context leaves (m, l, O) per query and run; a merge launch finishes the rows.
// PRE: the prefix before the window goes first, in key tiles of its own whose rows are counted from zero; its pages have a map of their own.
// All waits are bounded; a wait that runs out marks the launch failed, the roles keep their arrivals going, tensor memory is
// freed and the kernel returns.
#pragma once
#include <cuda.h>

#include <algorithm>
#include <map>
#include <mutex>

#include "attention_window_dev.cuh"
#include "tc05.cuh"

namespace {

constexpr int WT_QM = 128;
constexpr int WT_THREADS = 384;
// Registers: the block is launched with 168 a thread (384 x 168 = 64512).  The third warpgroup gives back all but 40, the
// softmax warpgroups grow to 232: 128 x 40 + 256 x 232 = 64512.
constexpr int WT_REGS_SMALL = 40, WT_REGS_LARGE = 232;
constexpr int WT_GROUP_MAX = 8;
constexpr int WT_TAB = 1344;  // floats of one bias table: eight heads x (16 rows + 127, padded)
constexpr int WT_TABLES = 21 * 1024;  // four of them
constexpr int WT_SMEM_CAP = 227 * 1024;
constexpr int WT_MAX_STAGES = 4;
constexpr uint32_t WT_COL_S = 0, WT_COL_O = 256, WT_TMEM = 512;  // scores of the two query tiles, then their outputs

template <int DK, int DV, int TN, bool KV>
struct WtGeo {
    static constexpr bool TABLES = DK <= 128;                     // wider keys leave no room for bias tables
    static constexpr int HEADER = 1024 + (TABLES ? WT_TABLES : 0);  // barriers; tables
    static constexpr int QTILE = WT_QM * DK * 2, V_AT = KV ? TN * DK * 2 : 0, STAGE = TN * DK * 2 + (KV ? TN * DV * 2 : 0);
    static constexpr int ROOM = (WT_SMEM_CAP - HEADER - 2 * QTILE) / STAGE;
    static constexpr int STAGES = ROOM < WT_MAX_STAGES ? ROOM : WT_MAX_STAGES;
    static constexpr size_t SMEM = (size_t)HEADER + 2 * QTILE + (size_t)STAGES * STAGE;
    static_assert(STAGES >= 2 && (KV || DK == DV), "");
};

struct WtBars {
    uint64_t kv_full[WT_MAX_STAGES], kv_empty[WT_MAX_STAGES], s_full[2], p_full[2], o_full[2];
    uint32_t tmem_base;
};

__device__ __forceinline__ void wt_g2s_2d(uint32_t dst_smem, const CUtensorMap* map, int x, int y, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst_smem),
                 "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(smem_u32(bar))
                 : "memory");
}
// byte offset of 16-byte chunk c of row r in a 128-byte-swizzled query tile: 64-column blocks of 128 rows x 128 bytes
__device__ __forceinline__ uint32_t wt_off(int r, int c) { return (uint32_t)((c >> 3) * (128 * 128) + r * 128 + (((c & 7) ^ (r & 7)) << 4)); }

__device__ __forceinline__ void st_32bytes(void* p, const uint32_t (&r)[8]) {  // one full sector per thread
    asm volatile("st.global.v8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"l"(p), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]),
                 "r"(r[7])
                 : "memory");
}

template <int DK, int DV, int TN, bool KV, bool PRE>
__global__ void __launch_bounds__(WT_THREADS, 1)
    window_attn_tc_kernel(const __grid_constant__ CUtensorMap kmap, int box_rows, const __grid_constant__ CUtensorMap pmap, int pre_box_rows, const __grid_constant__ WindowAttn a, const AttnTile* __restrict__ tiles,
                          int tiles_per_group, int rows_per_seq, int rows_per_tile, float* __restrict__ part_o, float2* __restrict__ part_ml,
                          uint32_t* __restrict__ err) {
    using Geo = WtGeo<DK, DV, TN, KV>;
    constexpr int STAGE = Geo::STAGE, QTILE = Geo::QTILE, WT_TN = TN, WT_STAGES = Geo::STAGES;
    extern __shared__ __align__(1024) uint8_t smem[];
    WtBars* bars = reinterpret_cast<WtBars*>(smem);
    float* tables = reinterpret_cast<float*>(smem + 1024);
    uint8_t* q_tiles = smem + Geo::HEADER;
    uint8_t* ring = q_tiles + 2 * QTILE;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kvh = blockIdx.y, n_splits = gridDim.x;
    const int grp = a.n_q_heads / a.keys.kv_heads;
    const int rows_wg = WT_QM / grp;            // rows of one query tile
    const int tile = (int)gridDim.z - 1 - (int)blockIdx.z;

    int row_first, n_rows;
    if (tiles) {
        row_first = tiles[tile].row_first, n_rows = tiles[tile].n_rows;
    } else {
        const int in_group = (tile % tiles_per_group) * rows_per_tile;
        row_first = (tile / tiles_per_group) * rows_per_seq + in_group;
        n_rows = min(rows_per_tile, rows_per_seq - in_group);
    }
    const tsb_row_desc rd0 = a.rows[row_first];
    const int seq = rd0.seq, pos0 = rd0.base + rd0.slot;
    const bool seq_ok = seq >= 0 && seq < a.keys.max_seqs && n_rows <= 2 * rows_wg;
    if (!seq_ok && threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
    if (!seq_ok) n_rows = 0;
    const int n_wg = n_rows > rows_wg ? 2 : 1;
    // visible positions, in key tiles that start at a copy box; this CTA's run of them
    const int lo = first_visible(a, pos0) & ~(box_rows - 1);
    const int hi = pos0 + n_rows;
    const int n_pre = PRE && seq_ok ? prefix_len(a, hi - 1) : 0, pre_tiles = (n_pre + WT_TN - 1) / WT_TN;
    const int total = seq_ok ? pre_tiles + (hi - lo + WT_TN - 1) / WT_TN : 0;
    const int per = (total + n_splits - 1) / n_splits;
    const int t_first = min(total, (int)blockIdx.x * per), n_tiles = min(total, t_first + per) - t_first;
    const int begin = lo + (t_first - pre_tiles) * WT_TN;  // of the window's tiles

    if (threadIdx.x == 0) {
        for (int i = 0; i < WT_STAGES; i++) mbar_init(&bars->kv_full[i], 1), mbar_init(&bars->kv_empty[i], 1);
        for (int i = 0; i < 2; i++) mbar_init(&bars->s_full[i], 1), mbar_init(&bars->p_full[i], 4), mbar_init(&bars->o_full[i], 1);
        mbar_fence_init();
    }
    if (warp == 9) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&bars->tmem_base)), "r"(WT_TMEM) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    pdl_wait();  // queries and this pass's keys come from the preceding kernel

    // ---- the query tiles, K-major, 128-byte swizzle
    for (int i = threadIdx.x; i < n_wg * WT_QM * (DK / 8); i += WT_THREADS) {
        const int x = i / (WT_QM * (DK / 8)), ql = (i / (DK / 8)) % WT_QM, c = i % (DK / 8);
        const int row = x * rows_wg + ql / grp;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (ql < rows_wg * grp && row < n_rows)
            v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(a.q) + (int64_t)(row_first + row) * a.q_stride +
                                                (kvh * grp + ql % grp) * DK + c * 8);
        *reinterpret_cast<uint4*>(q_tiles + x * QTILE + wt_off(ql, c)) = v;
    }
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bars->tmem_base;

    if (warp >= 8) {
        asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(WT_REGS_SMALL));
        if (warp == 8) {
            bool ok = true;
            int issued = 0;
            for (int t = 0; t < n_tiles && ok; t++) {
                const int st = t % WT_STAGES;
                if (t >= WT_STAGES && lane == 0) ok = mbar_wait(&bars->kv_empty[st], ((t / WT_STAGES) - 1) & 1, err);
                ok = __shfl_sync(0xffffffffu, (int)ok, 0) != 0;
                if (!ok) break;
                const uint32_t dst = smem_u32(ring + st * STAGE);
                if (lane == 0) mbar_expect_tx(&bars->kv_full[st], (uint32_t)STAGE);
                __syncwarp();
                const bool pre = PRE && t_first + t < pre_tiles, pooled = pre && a.pool > 0;
                const int box = pre ? pre_box_rows : box_rows, end = pre ? n_pre : hi, shift = pooled ? a.pooled.page_shift : a.keys.page_shift;
                const CUtensorMap* map = pre ? &pmap : &kmap;
                for (int part = lane; part * box < WT_TN; part += 32) {
                    int pos = (pre ? (t_first + t) * WT_TN : begin + t * WT_TN) + part * box;
                    if (pos >= end) pos = (end - 1) & ~(box - 1);  // past the end: masked later, read from a page that exists
                    const int lp = pos >> shift;
                    int page = lp < a.keys.max_pages_per_seq ? a.keys.page_table[(int64_t)seq * a.keys.max_pages_per_seq + lp] : -1;
                    if (page < 0) {  // not a reserved position: flagged; the copy reads page 0 so that the byte count stays whole
                        atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
                        page = 0;
                    }
                    const int row = (page << shift) + (pos & ((1 << shift) - 1));
#pragma unroll
                    for (int b = 0; b < DK / 64; b++)
                        wt_g2s_2d(dst + b * (WT_TN * 128) + part * box * 128, map, kvh * a.keys.head_step + b * 64, row, &bars->kv_full[st]);
                    if (KV) {
#pragma unroll
                        for (int b = 0; b < DV / 64; b++)
                            wt_g2s_2d(dst + Geo::V_AT + b * (WT_TN * 128) + part * box * 128, map, kvh * a.keys.head_step + a.keys.value_off + b * 64, row,
                                      &bars->kv_full[st]);
                    }
                }
                issued = t + 1;
                __syncwarp();
            }
            // no copy is in flight when the CTA leaves, also when another role has given up
            for (int t = lane > 0 ? issued : issued > WT_STAGES ? issued - WT_STAGES : 0; t < issued; t++) mbar_wait(&bars->kv_full[t % WT_STAGES], (t / WT_STAGES) & 1, err);
        }
        if (warp == 9) {
            const uint32_t leader = lane == 0 ? 1u : 0u;
            // f32 accumulate, bfloat16 operands, M = 128; scores: N = TN tokens, both operands K-major; output: N = DV, B MN-major
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(WT_QM >> 4) << 24);
            const uint32_t idesc_s = idesc | ((uint32_t)(WT_TN >> 3) << 17), idesc_o = idesc | (1u << 16) | ((uint32_t)(DV >> 3) << 17);
            constexpr uint64_t SW128 = 2ull << 61;
            const uint64_t kmaj = ((uint64_t)1u << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) | SW128;
            const uint64_t mnmaj = ((uint64_t)((uint32_t)(WT_TN * 128) >> 4) << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) | SW128;
            bool ok = true;
            auto scores = [&](int x, int t) {
                const uint64_t dq = kmaj | (uint64_t)((smem_u32(q_tiles + x * QTILE) >> 4) & 0x3FFFu);
                const uint64_t dk = kmaj | (uint64_t)((smem_u32(ring + (t % WT_STAGES) * STAGE) >> 4) & 0x3FFFu);
                const uint32_t d = tmem + WT_COL_S + (uint32_t)x * 128;
                tc_mma_ss<false>(leader, d, dq, dk, idesc_s);
#pragma unroll
                for (int ks = 1; ks < DK / 16; ks++) {
                    const uint64_t step = (uint64_t)((uint32_t)(ks & 3) * 2u);
                    tc_mma_ss<true>(leader, d, dq + (uint64_t)((uint32_t)(ks >> 2) * (128 * 128 / 16)) + step,
                                    dk + (uint64_t)((uint32_t)(ks >> 2) * (WT_TN * 128 / 16)) + step, idesc_s);
                }
                tc_commit_if(leader, &bars->s_full[x]);
            };
            if (n_tiles > 0) {
                ok = __all_sync(0xffffffffu, mbar_wait(&bars->kv_full[0], 0u, err));
                tc_fence_after();
                for (int x = 0; x < n_wg && ok; x++) scores(x, 0);
            }
            for (int t = 0; t < n_tiles && ok; t++) {
                const int st = t % WT_STAGES;
                const uint64_t dv = mnmaj | (uint64_t)((smem_u32(ring + st * STAGE + Geo::V_AT) >> 4) & 0x3FFFu);
                for (int x = 0; x < n_wg && ok; x++) {
                    ok = __all_sync(0xffffffffu, mbar_wait(&bars->p_full[x], t & 1, err));
                    if (!ok) break;
                    tc_fence_after();
                    const uint32_t d = tmem + WT_COL_O + (uint32_t)x * DV, p = tmem + WT_COL_S + (uint32_t)x * 128;  // P lies over the scores
                    if (t == 0) tc_mma_ts<false>(leader, d, p, dv, idesc_o);
                    else tc_mma_ts<true>(leader, d, p, dv, idesc_o);
#pragma unroll
                    for (int kt = 1; kt < WT_TN / 16; kt++) tc_mma_ts<true>(leader, d, p + 8 * kt, dv + (uint64_t)(128 * kt), idesc_o);
                    if (x == n_wg - 1) tc_commit_if(leader, &bars->kv_empty[st]);
                    if (t + 1 < n_tiles) {
                        if (x == 0) {
                            ok = __all_sync(0xffffffffu, mbar_wait(&bars->kv_full[(t + 1) % WT_STAGES], ((t + 1) / WT_STAGES) & 1, err));
                            tc_fence_after();
                        }
                        if (ok) scores(x, t + 1);  // in order behind the product that reads P from the same columns
                    } else {
                        tc_commit_if(leader, &bars->o_full[x]);
                    }
                }
            }
        }
    } else {
        asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(WT_REGS_LARGE));
        if (warp / 4 < n_wg) {
            // ---- softmax: thread = query ql of tile x = tensor-memory lane ql
            const int x = warp >> 2, ql = threadIdx.x & (WT_QM - 1);
            const int row_l = ql / grp, head_l = ql % grp;
            const int wg_first = pos0 + x * rows_wg, wg_last = min(wg_first + rows_wg, hi) - 1;  // positions of the tile's rows
            const bool valid = ql < rows_wg * grp && x * rows_wg + row_l < n_rows;
            const int pq = valid ? wg_first + row_l : -1;  // an empty slot sees nothing
            const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
            const uint32_t col_s = tmem + lane_base + WT_COL_S + (uint32_t)x * 128, col_o = tmem + lane_base + WT_COL_O + (uint32_t)x * DV;
            const bool capped = a.cap > 0.f, biased = Geo::TABLES && a.r1 != nullptr;
            const ScoreConst sc(a);
            const float slope = a.slopes ? a.slopes[kvh * grp + min(head_l, grp - 1)] * 1.4426950408889634f : 0.f;
            const int lo_last = first_visible(a, wg_last), lo_mine = first_visible(a, pq);
            const int pre_all = PRE ? prefix_len(a, wg_first) : 0, pre_mine = PRE ? prefix_len(a, pq) : 0;  // of the prefix: seen by every row, by this one
            // bias tables: entry k of a head holds the bias at distance wg_first - p0 + rows_wg - 1 - k; row_l's key j is entry
            // rows_wg - 1 - row_l + j.  The pitch keeps the 32 queries of a warp on different banks.
            const int need = rows_wg + WT_TN - 1;
            const int pitch = need + (((32 / grp) - need) & 31);
            float* tab[2] = {tables + (2 * x) * WT_TAB, tables + (2 * x + 1) * WT_TAB};
            const int tab_at = min(head_l, grp - 1) * pitch + max(rows_wg - 1 - row_l, 0);
            float m_ref = -INFINITY, l_run = 0.f;
            bool ok = true;
            for (int t = 0; t < n_tiles; t++) {
                const bool pre = PRE && t_first + t < pre_tiles;
                const int p0 = pre ? (t_first + t) * WT_TN : begin + t * WT_TN;
                const float* bias = tab[t & 1] + tab_at;
                if (biased) {
                    for (int h = 0; h < grp; h++) {
                        const float r1 = a.r1[kvh * grp + h], r2 = a.r2[kvh * grp + h];
                        for (int k = ql; k < need; k += WT_QM)
                            tab[t & 1][h * pitch + k] = -r1 * lg2(fmaf(r2, (float)max(wg_first - p0 + rows_wg - 1 - k, 0), 1.f));
                    }
                    asm volatile("bar.sync %0, 128;" ::"r"(1 + x) : "memory");
                }
                if (ok) ok = mbar_wait(&bars->s_full[x], t & 1, err);
                tc_fence_after();
                float s[WT_TN];
                {
                    uint32_t r[WT_TN / 16][16];
#pragma unroll
                    for (int c = 0; c < WT_TN / 16; c++) tc_ld16(col_s + 16 * c, r[c]);
                    tc_wait_ld();
#pragma unroll
                    for (int j = 0; j < WT_TN; j++) s[j] = __uint_as_float(r[j >> 4][j & 15]);
                }
                bool series = true;
                if (capped) {
                    float big = 0.f;
#pragma unroll
                    for (int j = 0; j < WT_TN; j++) big = fmaxf(big, fabsf(s[j]));
                    series = !__any_sync(0xffffffffu, big > sc.small);
                }
                if (capped && series) {
#pragma unroll
                    for (int j = 0; j < WT_TN; j += 2) {
                        const float2 x = make_float2(s[j], s[j + 1]), v = fma2(x, sc.factor(x), biased ? make_float2(bias[j], bias[j + 1]) : both(0.f));
                        s[j] = v.x, s[j + 1] = v.y;
                    }
                } else {
                    if (capped) {
#pragma unroll
                        for (int j = 0; j < WT_TN; j++) s[j] = fmaf(-2.f * sc.c_out, rcp(ex2(s[j] * sc.s_in) + 1.f), sc.c_out);
                    } else {
#pragma unroll
                        for (int j = 0; j < WT_TN; j++) s[j] *= sc.s_in;
                    }
                    if (biased) {
#pragma unroll
                        for (int j = 0; j < WT_TN; j++) s[j] += bias[j];
                    }
                }
                if (a.slopes) {
                    const float at0 = -slope * (float)(pq - p0);
#pragma unroll
                    for (int j = 0; j < WT_TN; j++) s[j] += fmaf(slope, (float)j, at0);
                }
                if (pre ? p0 + WT_TN > pre_all : p0 + WT_TN - 1 > wg_first || p0 < lo_last) {  // the tile meets an edge of some row
                    const int j_max = (pre ? pre_mine - 1 : pq) - p0, j_min = pre ? 0 : lo_mine - p0;
#pragma unroll
                    for (int j = 0; j < WT_TN; j++)
                        if (j > j_max || j < j_min) s[j] = -INFINITY;
                }
                float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
                for (int j = 0; j < WT_TN; j += 8) {
                    mx4[0] = max3(mx4[0], s[j], s[j + 1]), mx4[1] = max3(mx4[1], s[j + 2], s[j + 3]);
                    mx4[2] = max3(mx4[2], s[j + 4], s[j + 5]), mx4[3] = max3(mx4[3], s[j + 6], s[j + 7]);
                }
                const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
                const bool grow = mx > m_ref + 8.f;
                const float m_new = grow ? mx : m_ref;
                const float alpha = grow ? ex2(m_ref - m_new) : 1.f;  // 0 while nothing was visible
                if (__any_sync(0xffffffffu, grow && m_ref != -INFINITY)) {
                    // this tile's scores have arrived, so the products issued before them are complete
#pragma unroll
                    for (int c = 0; c < DV; c += 32) {
                        uint32_t r0[16], r1[16], w[32];
                        tc_ld16(col_o + c, r0);
                        tc_ld16(col_o + c + 16, r1);
                        tc_wait_ld();
#pragma unroll
                        for (int i = 0; i < 16; i++) w[i] = __float_as_uint(__uint_as_float(r0[i]) * alpha), w[16 + i] = __float_as_uint(__uint_as_float(r1[i]) * alpha);
                        tc_st32(col_o + c, w);
                    }
                }
                const float m_use = m_new == -INFINITY ? 0.f : m_new;
                float2 rs[2] = {both(0.f), both(0.f)};
#pragma unroll
                for (int c = 0; c < WT_TN; c += 64) {
                    uint32_t pk[32];
#pragma unroll
                    for (int j = 0; j < 64; j += 2) {
                        float2 e = add2(make_float2(s[c + j], s[c + j + 1]), both(-m_use));
                        e.x = ex2(e.x), e.y = ex2(e.y);
                        rs[(j >> 1) & 1] = add2(rs[(j >> 1) & 1], e);
                        pk[j >> 1] = pack_bf16(e.x, e.y);
                    }
                    tc_st32(col_s + (c >> 1), pk);
                }
                l_run = fmaf(l_run, alpha, (rs[0].x + rs[0].y) + (rs[1].x + rs[1].y));
                m_ref = m_new;
                tc_wait_st();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(&bars->p_full[x]);
            }
            if (ok && n_tiles > 0) ok = mbar_wait(&bars->o_full[x], 0u, err);
            tc_fence_after();
            const int row = row_first + x * rows_wg + row_l, head = kvh * grp + head_l;
            const int64_t share = (((int64_t)tile * a.keys.kv_heads + kvh) * n_splits + blockIdx.x) * (2 * WT_QM) + x * WT_QM + ql;
            float f = 0.f;
            if (valid && n_splits == 1) f = head_factor(a, row, head, m_ref, l_run);
#pragma unroll
            for (int c = 0; c < DV; c += 16) {
                float v[16];
                uint32_t r[16];
                if (n_tiles > 0) {  // the same for the whole warp
                    tc_ld16(col_o + c, r);
                    tc_wait_ld();
                }
#pragma unroll
                for (int i = 0; i < 16; i++) v[i] = n_tiles > 0 && ok ? __uint_as_float(r[i]) : 0.f;
                if (!valid) continue;
                if (n_splits == 1) {
                    if (a.turn) {
#pragma unroll
                        for (int i = 0; i < 16; i += 2) turn_back(a, row, c + i, v[i], v[i + 1]);
                    }
                    if (a.value_gate) {
                        const uint4* g = reinterpret_cast<const uint4*>(value_gate_at(a, row, head, c));
#pragma unroll
                        for (int h = 0; h < 2; h++) {
                            const uint4 z = g[h];
                            const uint32_t zz[4] = {z.x, z.y, z.z, z.w};
#pragma unroll
                            for (int i = 0; i < 4; i++)
                                v[8 * h + 2 * i] *= rcp(1.f + ex2(__uint_as_float(zz[i] << 16) * -1.4426950408889634f)),
                                    v[8 * h + 2 * i + 1] *= rcp(1.f + ex2(__uint_as_float(zz[i] & 0xFFFF0000u) * -1.4426950408889634f));
                        }
                    }
                    uint32_t w[8];
#pragma unroll
                    for (int i = 0; i < 8; i++) w[i] = pack_bf16(v[2 * i] * f, v[2 * i + 1] * f);
                    st_32bytes(reinterpret_cast<__nv_bfloat16*>(a.out) + (int64_t)row * a.out_stride + head * DV + c, w);
                } else {
                    uint32_t w[8];
#pragma unroll
                    for (int h = 0; h < 2; h++) {
#pragma unroll
                        for (int i = 0; i < 8; i++) w[i] = __float_as_uint(v[8 * h + i]);
                        st_32bytes(part_o + share * DV + c + 8 * h, w);
                    }
                }
            }
            if (valid && n_splits > 1) part_ml[share] = make_float2(m_ref, l_run);
        }
    }
    pdl_launch_dependents();
    tc_fence_before();
    __syncthreads();
    if (warp == 9) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(WT_TMEM) : "memory");
    }
}

// 2-D bfloat16 map over the token rows of a layer's pages, box 64 columns x box_rows rows, 128-byte swizzle; kept per
// (address, shape).  Encoding goes through the driver entry point (no link against libcuda).
cudaError_t wt_map(const KeyView& k, int box_rows, CUtensorMap* out) {
    typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                 const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
    static std::mutex mu;
    static EncodeFn encode = nullptr;
    struct Key {
        const void* p;
        int64_t rows;
        int cols, box;
        bool operator<(const Key& o) const {
            return p != o.p ? p < o.p : rows != o.rows ? rows < o.rows : cols != o.cols ? cols < o.cols : box < o.box;
        }
    };
    static std::map<Key, CUtensorMap> cache;
    std::lock_guard<std::mutex> lock(mu);
    if (!encode) {
        void* fn = nullptr;
        cudaDriverEntryPointQueryResult qres;
        cudaError_t e = cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres);
        if (e != cudaSuccess) return e;
        if (!fn || qres != cudaDriverEntryPointSuccess) return cudaErrorNotSupported;
        encode = reinterpret_cast<EncodeFn>(fn);
    }
    const Key key{k.base, (int64_t)k.num_pages * k.page_tokens, k.row, box_rows};
    auto it = cache.find(key);
    if (it == cache.end()) {
        if (cache.size() > 8192) cache.clear();
        CUtensorMap m;
        const cuuint64_t gdim[2] = {(cuuint64_t)key.cols, (cuuint64_t)key.rows};
        const cuuint64_t gstride[1] = {(cuuint64_t)key.cols * 2};
        const cuuint32_t box[2] = {64, (cuuint32_t)box_rows};
        const cuuint32_t estride[2] = {1, 1};
        if (encode(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, k.base, gdim, gstride, box, estride, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                   CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
            return cudaErrorInvalidValue;
        it = cache.emplace(key, m).first;
    }
    *out = it->second;
    return cudaSuccess;
}

template <int DK, int DV, int TN, bool KV, bool PRE = false>
cudaError_t launch_tc(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    const int splits = wattn_splits(ctx, a, l, TN, 2 * WT_QM, 1);
    const WattnScratch sc = wattn_scratch(ctx, scratch);
    const int box_rows = std::min(a.keys.page_tokens, TN);
    CUtensorMap map;
    if (cudaError_t e = wt_map(a.keys, box_rows, &map); e != cudaSuccess) return e;
    const KeyView& prefix = a.pool > 0 ? a.pooled : a.keys;
    const int pre_box_rows = std::min(prefix.page_tokens, TN);
    CUtensorMap pmap = map;
    if (PRE)
        if (cudaError_t e = wt_map(prefix, pre_box_rows, &pmap); e != cudaSuccess) return e;
    static SmemOptIn configured;
    constexpr size_t smem = WtGeo<DK, DV, TN, KV>::SMEM;
    if (cudaError_t e = tsb_opt_in_smem(ctx, window_attn_tc_kernel<DK, DV, TN, KV, PRE>, smem, configured); e != cudaSuccess) return e;
    cudaError_t e = tsb_launch(ctx, window_attn_tc_kernel<DK, DV, TN, KV, PRE>, dim3((unsigned)splits, (unsigned)a.keys.kv_heads, (unsigned)l.n_tiles),
                               dim3(WT_THREADS), smem, st, true, map, box_rows, pmap, pre_box_rows, a, l.tiles, l.tiles_per_group, l.rows_per_seq, l.rows_per_tile, sc.o, sc.ml,
                               ctx->dev_error);
    return e == cudaSuccess && splits > 1 ? launch_window_attn_merge(ctx, st, a, l, splits, 2 * WT_QM, sc) : e;
}

}  // namespace
