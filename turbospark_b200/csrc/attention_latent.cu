// Attention over latent rows (attention_latent.cuh), bfloat16, mma.sync m16n8k16.
//
// A CTA owns a query tile - 16 MT (row, head) pairs of one stream - and a run of 64-token key tiles, fetched row by row with
// bulk copies into a ring of stages.  One tile in shared memory serves both products, and a key byte is read from memory once.
// Eight warps:
//   scores   KS warps split the key columns, 8 / KS groups of them the keys; a warp's part of every query stays in registers, so this
//            product reads each key fragment once and nothing else.  The parts meet in shared memory.
//   softmax  256 / (16 MT) threads per query add the parts, mask, keep the running maximum and sum, leave the weights (bfloat16)
//            and the factor of the earlier sums
//   output   every warp owns DV / 8 value columns of all queries
// so the accumulators of a 512-column value fit in registers.  Key tiles start at multiples of 64 positions.  A context that does
// not fill the device with CTAs is cut into runs; a merge launch adds them in order.
// Waits for copies are bounded; when one runs out the launch is marked failed and the warps go on meeting until the end, where the
// CTA waits (again with a limit) for what it has in flight.
#include <algorithm>

#include "attention_latent.cuh"
#include "attention_window_dev.cuh"

namespace {

constexpr int LT_TOK = 64, LT_WARPS = 8, LT_THREADS = LT_WARPS * 32;
constexpr int LT_SMEM_CAP = 227 * 1024;
constexpr int LT_P_PITCH = LT_TOK * 2 + 16;    // bytes
constexpr int LT_S_PITCH = LT_TOK + 8;         // floats
constexpr int LT_HEADER = 128;                 // barriers

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm2_t(uint32_t& r0, uint32_t& r1, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// DV value columns, key columns in KW blocks of 64, MT query tiles of sixteen.
template <int DV, int KW, int MT>
struct LtGeo {
    static constexpr int KS = DV > 128 ? 4 : 2, GROUPS = LT_WARPS / KS, KEYS = LT_TOK / GROUPS;  // keys of a warp's scores
    static constexpr int STEPS = KW * 4 / KS;                                                  // sixteen-column steps of a warp's part
    static constexpr int PITCH = KW * 128 + 16;  // bytes of a key row: eight rows of a chunk meet all banks
    static constexpr int STAGES = DV > 256 ? 2 : 3, STAGE = LT_TOK * PITCH, QT = 16 * MT;
    static constexpr size_t SMEM = (size_t)LT_HEADER + STAGES * STAGE + (size_t)KS * QT * LT_S_PITCH * 4 + QT * (LT_P_PITCH + 8);
    static constexpr int PER_SM = DV <= 128 ? 2 : 1;
};

template <int DV, int KW, int MT>
__global__ void __launch_bounds__(LT_THREADS, LtGeo<DV, KW, MT>::PER_SM)
    latent_attn_kernel(const __grid_constant__ LatentAttn a, const AttnTile* __restrict__ tiles, int tiles_per_group, int rows_per_seq, int rows_per_tile,
                       int heads_per_tile, float* __restrict__ part_o, float2* __restrict__ part_ml, uint32_t* __restrict__ err) {
    using G = LtGeo<DV, KW, MT>;
    constexpr int QT = G::QT, NST = G::STAGES, KS = G::KS, NT = G::KEYS / 8;
    constexpr int ND = DV / 64;                                       // n-tiles of eight value columns per warp
    constexpr int TPQ = LT_THREADS / QT, PER = LT_TOK / TPQ;            // threads per query, scores per thread
    extern __shared__ __align__(128) uint8_t smem[];
    uint64_t* full = reinterpret_cast<uint64_t*>(smem);
    uint8_t* ring = smem + LT_HEADER;
    float* parts = reinterpret_cast<float*>(ring + NST * G::STAGE);                   // [KS][QT][LT_S_PITCH]
    uint8_t* p_tile = reinterpret_cast<uint8_t*>(parts + KS * QT * LT_S_PITCH);       // [QT], bfloat16
    float* alphas = reinterpret_cast<float*>(p_tile + QT * LT_P_PITCH);               // [QT]; the sums at the end
    float* maxima = alphas + QT;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int kq = warp % KS, kg = warp / KS;
    const int n_splits = gridDim.x, DK = a.keys.head_dim;
    int row_first, n_rows;
    if (tiles) {
        row_first = tiles[blockIdx.z].row_first, n_rows = tiles[blockIdx.z].n_rows;
    } else {
        const int in_group = ((int)blockIdx.z % tiles_per_group) * rows_per_tile;
        row_first = ((int)blockIdx.z / tiles_per_group) * rows_per_seq + in_group;
        n_rows = min(rows_per_tile, rows_per_seq - in_group);
    }
    const tsb_row_desc rd0 = a.rows[row_first];
    const int seq = rd0.seq, pos0 = rd0.base + rd0.slot;
    const int head0 = blockIdx.y * heads_per_tile, heads = min(heads_per_tile, a.n_heads - head0);
    const int n_queries = n_rows * heads;
    if (seq < 0 || seq >= a.keys.max_seqs || n_queries > QT || DK > KW * 64) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        pdl_wait();
        return;
    }
    const int hi = pos0 + n_rows;
    const int total = (hi + LT_TOK - 1) / LT_TOK, per = (total + n_splits - 1) / n_splits;
    const int t_first = min(total, (int)blockIdx.x * per), n_tiles = min(total, t_first + per) - t_first;
    const int begin = t_first * LT_TOK;
    const uint32_t ring_s = smem_u32(ring), p_smem = smem_u32(p_tile);

    if (threadIdx.x == 0) {
        for (int i = 0; i < NST; i++) mbar_init(&full[i], LT_WARPS);
        mbar_fence_init();
    }
    // columns behind the row's: finite, and the queries have zeros there
    for (int i = threadIdx.x; i < NST * LT_TOK * (KW * 8 - DK / 8); i += LT_THREADS) {
        const int r = i / (KW * 8 - DK / 8), c = DK / 8 + i % (KW * 8 - DK / 8);
        *reinterpret_cast<uint4*>(ring + (size_t)r * G::PITCH + c * 16) = make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
    // Every warp fetches eight rows of a tile, a lane each.  Positions past the end are masked later; their slots repeat the last row.
    // The row's address is looked up a tile ahead.
    auto row_of = [&](int tile) -> const __nv_bfloat16* {
        if (lane >= 8 || tile >= n_tiles) return nullptr;
        const __nv_bfloat16* src = key_row<__nv_bfloat16>(a.keys, seq, min(begin + tile * LT_TOK + warp * 8 + lane, hi - 1));
        if (src) return src;
        atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);  // not a reserved position: flagged; the copy keeps its byte count
        return reinterpret_cast<const __nv_bfloat16*>(a.keys.base);
    };
    auto issue = [&](int tile, const __nv_bfloat16* src) {
        if (tile >= n_tiles) return;
        uint64_t* bar = &full[tile % NST];
        if (lane == 0) mbar_expect_tx(bar, (uint32_t)(8 * DK * 2));
        __syncwarp();
        if (lane < 8) bulk_g2s(ring + (size_t)((tile % NST) * LT_TOK + warp * 8 + lane) * G::PITCH, src, (uint32_t)(DK * 2), bar);
    };
    const bool early = begin + (NST - 1) * LT_TOK <= rd0.base;  // keys of earlier passes
    if (!early) pdl_wait();
#pragma unroll
    for (int i = 0; i < NST - 1; i++) issue(i, row_of(i));
    const __nv_bfloat16* next_row = row_of(NST - 1);
    if (early) pdl_wait();
    // this warp's part of the queries
    uint32_t qf[MT][G::STEPS][4];
#pragma unroll
    for (int m = 0; m < MT; m++) {
        const uint32_t* qp[2];
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int qi = m * 16 + gid + 8 * h;
            qp[h] = qi < n_queries ? reinterpret_cast<const uint32_t*>(static_cast<const __nv_bfloat16*>(a.q) + (int64_t)(row_first + qi / heads) * a.q_stride +
                                                                      (int64_t)(head0 + qi % heads) * DK)
                                   : nullptr;
        }
#pragma unroll
        for (int k = 0; k < G::STEPS; k++) {
            const int c = (kq * G::STEPS + k) * 16;
#pragma unroll
            for (int i = 0; i < 4; i++) qf[m][k][i] = qp[i & 1] && c < DK ? qp[i & 1][c / 2 + (i >> 1) * 4 + tig] : 0u;
        }
    }
    // the thread's query of the softmax
    const int sq = threadIdx.x / TPQ, sj = threadIdx.x % TPQ;
    const int pq = pos0 + (sq < n_queries ? sq / heads : 0);  // an empty slot repeats the first query and is not stored
    const float scale2 = a.scale * 1.4426950408889634f;
    float m_run = -INFINITY, l_run = 0.f;
    float o[MT][ND][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int n = 0; n < ND; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) o[m][n][i] = 0.f;
    const int col0 = warp * (DV / LT_WARPS);
    bool ok = true;

    for (int tile = 0; tile < n_tiles; tile++) {
        // the tile is here, and every warp is done with the stage and the weights of the one before
        if (ok) ok = mbar_wait(&full[tile % NST], (tile / NST) & 1, err);  // a wait that ran out: the launch is marked, its result void
        __syncthreads();
        issue(tile + NST - 1, next_row);
        next_row = row_of(tile + NST);
        const uint32_t kt = ring_s + (tile % NST) * G::STAGE;
        float s[MT][NT][4];
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int n = 0; n < NT; n++)
#pragma unroll
                for (int i = 0; i < 4; i++) s[m][n][i] = 0.f;
        const uint32_t ka = kt + (kg * G::KEYS + (lane & 7) + ((lane >> 4) << 3)) * G::PITCH + kq * G::STEPS * 32 + ((lane >> 3) & 1) * 16;
#pragma unroll
        for (int k = 0; k < G::STEPS; k++) {
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                uint32_t b[4];
                ldsm4(b, ka + n * 8 * G::PITCH + k * 32);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    mma_bf16(s[m][n], qf[m][k], b[0], b[1]);
                    mma_bf16(s[m][n + 1], qf[m][k], b[2], b[3]);
                }
            }
        }
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int n = 0; n < NT; n++) {
                float* d = parts + (kq * QT + m * 16 + gid) * LT_S_PITCH + kg * G::KEYS + n * 8 + 2 * tig;
                *reinterpret_cast<float2*>(d) = make_float2(s[m][n][0], s[m][n][1]);
                *reinterpret_cast<float2*>(d + 8 * LT_S_PITCH) = make_float2(s[m][n][2], s[m][n][3]);
            }
        __syncthreads();
        {
            const int p0 = begin + tile * LT_TOK;
            float v[PER];
            float mx = -INFINITY;
#pragma unroll
            for (int c = 0; c < PER; c += 4) {
                const int col = (c / 4 * TPQ + sj) * 4;
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int k = 0; k < KS; k++) {
                    const float4 y = *reinterpret_cast<const float4*>(parts + (k * QT + sq) * LT_S_PITCH + col);
                    x.x += y.x, x.y += y.y, x.z += y.z, x.w += y.w;
                }
                const float xs[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    v[c + i] = p0 + col + i <= pq ? xs[i] * scale2 : -INFINITY;
                    mx = fmaxf(mx, v[c + i]);
                }
            }
#pragma unroll
            for (int d = TPQ / 2; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
            const float m_new = fmaxf(m_run, mx), use = m_new == -INFINITY ? 0.f : m_new;
            const float alpha = ex2(m_run - use);  // 0 while nothing was visible
            m_run = m_new;
            float sum = 0.f;
#pragma unroll
            for (int c = 0; c < PER; c += 4) {
                const int col = (c / 4 * TPQ + sj) * 4;
#pragma unroll
                for (int i = 0; i < 4; i++) v[c + i] = ex2(v[c + i] - use), sum += v[c + i];
                *reinterpret_cast<uint2*>(p_tile + sq * LT_P_PITCH + col * 2) = make_uint2(pack_bf16(v[c], v[c + 1]), pack_bf16(v[c + 2], v[c + 3]));
            }
            l_run = fmaf(l_run, alpha, sum);
            if (sj == 0) alphas[sq] = alpha;
        }
        __syncthreads();
        float al[MT][2];
        bool moved = false;
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int h = 0; h < 2; h++) al[m][h] = alphas[m * 16 + gid + 8 * h], moved |= al[m][h] != 1.f;
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int n = 0; n < ND; n++) o[m][n][0] *= al[m][0], o[m][n][1] *= al[m][0], o[m][n][2] *= al[m][1], o[m][n][3] *= al[m][1];
        }
#pragma unroll
        for (int kk = 0; kk < LT_TOK / 16; kk++) {
            uint32_t pa[MT][4];
#pragma unroll
            for (int m = 0; m < MT; m++) ldsm4(pa[m], p_smem + (m * 16 + (lane & 15)) * LT_P_PITCH + kk * 32 + (lane >> 4) * 16);
            const uint32_t va = kt + (kk * 16 + (lane & 15)) * G::PITCH + col0 * 2;
#pragma unroll
            for (int np = 0; np < ND / 2; np++) {
                uint32_t b[4];
                ldsm4_t(b, va + np * 32 + (lane >> 4) * 16);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    mma_bf16(o[m][2 * np], pa[m], b[0], b[1]);
                    mma_bf16(o[m][2 * np + 1], pa[m], b[2], b[3]);
                }
            }
            if (ND & 1) {
                uint32_t b0, b1;
                ldsm2_t(b0, b1, va + (ND / 2) * 32);
#pragma unroll
                for (int m = 0; m < MT; m++) mma_bf16(o[m][ND - 1], pa[m], b0, b1);
            }
        }
        }
    if (!ok)  // no copy is in flight when the CTA leaves
        for (int i = max(0, n_tiles - NST); i < n_tiles; i++) mbar_wait(&full[i % NST], (i / NST) & 1, err);
    pdl_launch_dependents();
    __syncthreads();
#pragma unroll
    for (int d = TPQ / 2; d > 0; d >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, d);
    if (sj == 0) alphas[sq] = l_run, maxima[sq] = m_run;
    __syncthreads();
    const int64_t tile_id = (int64_t)blockIdx.z * gridDim.y + blockIdx.y;
    const int64_t share = (tile_id * n_splits + blockIdx.x) * QT;
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int qi = m * 16 + gid + 8 * h;
            if (qi >= n_queries) continue;
            const float l = alphas[qi], mx = maxima[qi];
            const int head = head0 + qi % heads;
            if (n_splits == 1) {
                const float f = 1.f / (a.sink ? l + ex2(a.sink[head] * 1.4426950408889634f - mx) : l);
                __nv_bfloat16* p = static_cast<__nv_bfloat16*>(a.out) + (int64_t)(row_first + qi / heads) * a.out_stride + (int64_t)head * DV + col0;
#pragma unroll
                for (int n = 0; n < ND; n++) *reinterpret_cast<uint32_t*>(p + n * 8 + 2 * tig) = pack_bf16(o[m][n][2 * h] * f, o[m][n][2 * h + 1] * f);
            } else {
                float* p = part_o + (share + qi) * DV + col0;
#pragma unroll
                for (int n = 0; n < ND; n++) *reinterpret_cast<float2*>(p + n * 8 + 2 * tig) = make_float2(o[m][n][2 * h], o[m][n][2 * h + 1]);
                if (warp == 0 && tig == 0) part_ml[share + qi] = make_float2(mx, l);
            }
        }
}

// One CTA per query slot of a tile: warps over 128-column pieces, the runs' weights in the lanes.
__global__ void __launch_bounds__(128)
    latent_merge_kernel(const __grid_constant__ LatentAttn a, const AttnTile* __restrict__ tiles, int tiles_per_group, int rows_per_seq, int rows_per_tile,
                        int heads_per_tile, int n_splits, int slots, const float* __restrict__ part_o, const float2* __restrict__ part_ml) {
    const int qi = blockIdx.x, tile = blockIdx.z;
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
    const int head0 = blockIdx.y * heads_per_tile, heads = min(heads_per_tile, a.n_heads - head0);
    if (qi >= n_rows * heads) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = head0 + qi % heads, DV = a.value_dim;
    const int64_t first = ((int64_t)tile * gridDim.y + blockIdx.y) * n_splits * slots + qi;
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
#pragma unroll
    for (int i = 0; i < WATTN_MAX_SPLITS / 32; i++) v[i].x = ex2(v[i].x - m), l = fmaf(v[i].y, v[i].x, l);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
    if (a.sink) l += ex2(a.sink[head] * 1.4426950408889634f - m);
    const float f = 1.f / l;
    for (int c0 = warp * 128; c0 < DV; c0 += 512) {
        const int c = c0 + lane * 4;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int k = 0; k < n_splits; k++) {
            const float w = __shfl_sync(0xffffffffu, k < 32 ? v[0].x : v[1].x, k & 31);
            if (c < DV) {
                const float4 x = *reinterpret_cast<const float4*>(part_o + (first + (int64_t)k * slots) * DV + c);
                acc.x = fmaf(x.x, w, acc.x), acc.y = fmaf(x.y, w, acc.y), acc.z = fmaf(x.z, w, acc.z), acc.w = fmaf(x.w, w, acc.w);
            }
        }
        if (c < DV)
            *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(a.out) + (int64_t)(row_first + qi / heads) * a.out_stride + (int64_t)head * DV + c) =
                make_uint2(pack_bf16(acc.x * f, acc.y * f), pack_bf16(acc.z * f, acc.w * f));
    }
}

template <int DV, int KW, int MT>
cudaError_t launch_one(tsb_ctx* ctx, cudaStream_t st, const LatentAttn& a, const WattnLaunch& l, int heads_per_tile, void* scratch) {
    using G = LtGeo<DV, KW, MT>;
    const int head_tiles = (a.n_heads + heads_per_tile - 1) / heads_per_tile, base = l.n_tiles * head_tiles;
    const int splits = wattn_splits(ctx, 0, l, LT_TOK, G::QT, G::PER_SM, base, std::min(wattn_part_queries(ctx), wattn_part_queries(ctx) * 256 / DV));
    const WattnScratch sc = wattn_scratch(ctx, scratch);
    static SmemOptIn configured;
    static_assert(G::SMEM <= (size_t)LT_SMEM_CAP, "");
    if (cudaError_t e = tsb_opt_in_smem(ctx, latent_attn_kernel<DV, KW, MT>, G::SMEM, configured); e != cudaSuccess) return e;
    cudaError_t e = tsb_launch(ctx, latent_attn_kernel<DV, KW, MT>, dim3((unsigned)splits, (unsigned)head_tiles, (unsigned)l.n_tiles), dim3(LT_THREADS),
                               G::SMEM, st, true, a, l.tiles, l.tiles_per_group, l.rows_per_seq, l.rows_per_tile, heads_per_tile, sc.o, sc.ml, ctx->dev_error);
    if (e == cudaSuccess && splits > 1)
        e = tsb_launch(ctx, latent_merge_kernel, dim3(G::QT, (unsigned)head_tiles, (unsigned)l.n_tiles), dim3(128), 0, st, true, a, l.tiles, l.tiles_per_group,
                       l.rows_per_seq, l.rows_per_tile, heads_per_tile, splits, G::QT, (const float*)sc.o, (const float2*)sc.ml);
    return e;
}
template <int DV>
cudaError_t launch_dim(tsb_ctx* ctx, cudaStream_t st, const LatentAttn& a, const WattnLaunch& l, const LatentTiling& t, void* scratch) {
    constexpr int KW = DV / 64 + 1;
    if (a.keys.head_dim <= KW * 64)
        return t.queries == 16 ? launch_one<DV, KW, 1>(ctx, st, a, l, t.heads, scratch) : launch_one<DV, KW, 2>(ctx, st, a, l, t.heads, scratch);
    return t.queries == 16 ? launch_one<DV, KW + 1, 1>(ctx, st, a, l, t.heads, scratch) : launch_one<DV, KW + 1, 2>(ctx, st, a, l, t.heads, scratch);
}

}  // namespace

bool latent_attn_dims(int kv_rank, int rot_dim, int* key_dim, int* value_dim) {
    for (int dv : {64, 128, 192, 256, 384, 512}) {
        if (kv_rank > dv) continue;
        const int dk = std::max((kv_rank + rot_dim + 31) / 32 * 32, dv);
        if (dk > dv + 128) return false;
        *key_dim = dk, *value_dim = dv;
        return true;
    }
    return false;
}

LatentTiling latent_attn_tiling(const tsb_ctx* ctx, int n_heads, int most_rows, int n_rows, int max_len) {
    LatentTiling t;
    // sixteen queries a tile where 32 would leave SMs idle: the key tiles of few streams
    const int64_t work = (int64_t)((n_rows * (int64_t)n_heads + 31) / 32) * ((max_len + LT_TOK - 1) / LT_TOK);
    t.queries = n_heads * most_rows <= 16 || work < ctx->sm_count ? 16 : 32;
    const int head_tiles = (n_heads + t.queries - 1) / t.queries;
    t.heads = (n_heads + head_tiles - 1) / head_tiles;
    t.rows = std::max(1, std::min(most_rows, t.queries / t.heads));
    return t;
}

cudaError_t launch_latent_attn(tsb_ctx* ctx, cudaStream_t st, const LatentAttn& a, const AttnBatch& b, const LatentTiling& t, void* scratch) {
    WattnLaunch l{b.small, b.n_small, 1, 0, t.rows, b.max_len};
    if (b.rows_per_seq > 0) {
        const int tpg = (b.rows_per_seq + t.rows - 1) / t.rows;
        l = WattnLaunch{nullptr, b.rows / b.rows_per_seq * tpg, tpg, b.rows_per_seq, t.rows, b.max_len};
    }
    if (l.n_tiles == 0) return cudaSuccess;
    switch (a.value_dim) {
        case 64: return launch_dim<64>(ctx, st, a, l, t, scratch);
        case 128: return launch_dim<128>(ctx, st, a, l, t, scratch);
        case 192: return launch_dim<192>(ctx, st, a, l, t, scratch);
        case 256: return launch_dim<256>(ctx, st, a, l, t, scratch);
        case 384: return launch_dim<384>(ctx, st, a, l, t, scratch);
        case 512: return launch_dim<512>(ctx, st, a, l, t, scratch);
        default: return cudaErrorInvalidValue;
    }
}
