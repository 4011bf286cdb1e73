// Attention over latent rows (attention_latent.cuh), bfloat16, mma.sync m16n8k16.
//
// A CTA owns a query tile - 16 MT (row, head) pairs of one stream - and a run of 64-token key tiles, which cp.async brings into a
// ring of row-padded stages.  One tile in shared memory serves both products.  Eight warps:
//   scores   MT warps share a group of 8 MT keys, each with sixteen of the queries; all of them walk the whole key width
//   softmax  row maxima of the key groups meet in shared memory; every warp keeps the running maximum of every query
//   output   every warp owns DV / 8 value columns of all queries; the weights come from shared memory
// so the accumulators of a 512-column value fit in registers and a key byte is read from memory once.  Key tiles start at
// multiples of 64 positions.  A context that does not fill the device with CTAs is cut into runs; a merge launch adds them in order.
#include <algorithm>

#include "attention_latent.cuh"
#include "attention_window_dev.cuh"

namespace {

constexpr int LT_TOK = 64, LT_WARPS = 8, LT_THREADS = LT_WARPS * 32;
constexpr int LT_SMEM_CAP = 227 * 1024;
constexpr int LT_P_PITCH = LT_TOK * 2 + 16;

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
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}

__host__ __device__ constexpr int lt_pitch(int key_dim) { return key_dim * 2 + 16; }  // key_dim a multiple of 32: eight rows of a chunk meet all banks
template <int DV>
constexpr int lt_stages() { return DV > 256 ? 2 : 3; }
template <int DV, int MT>
size_t lt_smem(int key_dim) {
    return (size_t)(lt_stages<DV>() * LT_TOK + 16 * MT) * lt_pitch(key_dim) + 16 * MT * (LT_P_PITCH + LT_WARPS * 4);
}
constexpr int lt_per_sm(int dv, int mt) { return dv <= 128 ? 2 : dv <= 256 && mt <= 2 ? 2 : 1; }

template <int DV, int MT>
__global__ void __launch_bounds__(LT_THREADS, lt_per_sm(DV, MT))
    latent_attn_kernel(const __grid_constant__ LatentAttn a, const AttnTile* __restrict__ tiles, int tiles_per_group, int rows_per_seq, int rows_per_tile,
                       int heads_per_tile, float* __restrict__ part_o, float2* __restrict__ part_ml, uint32_t* __restrict__ err) {
    constexpr int QT = 16 * MT, NG = LT_WARPS / MT, NK = MT, NST = lt_stages<DV>();  // key groups; n-tiles of eight keys per warp
    constexpr int ND = DV / 64;                                                      // n-tiles of eight value columns per warp
    extern __shared__ __align__(128) uint8_t smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int mt = warp % MT, kg = warp / MT;
    const int n_splits = gridDim.x, DK = a.keys.head_dim, pitch = lt_pitch(DK);
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
    if (seq < 0 || seq >= a.keys.max_seqs || n_queries > QT) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        pdl_wait();
        return;
    }
    const int hi = pos0 + n_rows;
    const int total = (hi + LT_TOK - 1) / LT_TOK, per = (total + n_splits - 1) / n_splits;
    const int t_first = min(total, (int)blockIdx.x * per), n_tiles = min(total, t_first + per) - t_first;
    const int begin = t_first * LT_TOK;

    uint8_t* q_tile = smem + (size_t)NST * LT_TOK * pitch;
    uint8_t* p_tile = q_tile + QT * pitch;
    float* group_max = reinterpret_cast<float*>(p_tile + QT * LT_P_PITCH);  // [QT][NG]; the groups' sums at the end
    const uint32_t ring = smem_u32(smem), q_smem = smem_u32(q_tile), p_smem = smem_u32(p_tile);

    auto issue = [&](int tile) {
        if (tile < n_tiles) {
            // four threads a token row
            const int r = threadIdx.x >> 2, pos = begin + tile * LT_TOK + r;
            const __nv_bfloat16* src = pos < hi ? key_row<__nv_bfloat16>(a.keys, seq, pos) : nullptr;
            const bool ok = src != nullptr;
            if (!ok) src = reinterpret_cast<const __nv_bfloat16*>(a.keys.base);
            const uint32_t dst = ring + (tile % NST) * LT_TOK * pitch + r * pitch;
            for (int c = threadIdx.x & 3; c < DK / 8; c += 4) cp16(dst + c * 16, ok ? src + c * 8 : src, ok);
        }
        cp_async_commit();
    };
    const bool early = begin + (NST - 1) * LT_TOK <= rd0.base;  // keys of earlier passes
    if (early) {
#pragma unroll
        for (int i = 0; i < NST - 1; i++) issue(i);
    }
    pdl_wait();
    if (!early) {
#pragma unroll
        for (int i = 0; i < NST - 1; i++) issue(i);
    }
    for (int i = threadIdx.x; i < QT * (DK / 8); i += LT_THREADS) {
        const int qi = i / (DK / 8), c = i % (DK / 8);
        uint4 v = make_uint4(0, 0, 0, 0);
        if (qi < n_queries)
            v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.q) + (int64_t)(row_first + qi / heads) * a.q_stride +
                                                (int64_t)(head0 + qi % heads) * DK + c * 8);
        *reinterpret_cast<uint4*>(q_tile + qi * pitch + c * 16) = v;
    }
    // positions of the lane's two score rows; empty slots repeat the first query and are not stored
    int pq[2];
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int qi = mt * 16 + gid + 8 * h;
        pq[h] = pos0 + (qi < n_queries ? qi / heads : 0);
    }
    const float scale2 = a.scale * 1.4426950408889634f;
    float o[MT][ND][4];
    float m_run[MT][2], l_run[2] = {0.f, 0.f};
#pragma unroll
    for (int m = 0; m < MT; m++) {
        m_run[m][0] = m_run[m][1] = -INFINITY;
#pragma unroll
        for (int n = 0; n < ND; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) o[m][n][i] = 0.f;
    }
    const int col0 = warp * (DV / LT_WARPS);

    for (int tile = 0; tile < n_tiles; tile++) {
        cp_async_wait<NST - 2>();
        __syncthreads();  // the tile is here, and every warp is done with the stage and the weights of the one before
        issue(tile + NST - 1);
        const uint32_t kt = ring + (tile % NST) * LT_TOK * pitch;
        const int key0 = kg * 8 * NK;
        float s[NK][4], s2[NK][4];
#pragma unroll
        for (int n = 0; n < NK; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) s[n][i] = 0.f, s2[n][i] = 0.f;
        const uint32_t qa = q_smem + (mt * 16 + (lane & 15)) * pitch + (lane >> 4) * 16;
        const uint32_t ka = kt + (key0 + (lane & 7)) * pitch + (lane >> 3) * 16;
#pragma unroll 2
        for (int kp = 0; kp < DK / 32; kp++) {
            uint32_t a0[4], a1[4];
            ldsm4(a0, qa + kp * 64);
            ldsm4(a1, qa + kp * 64 + 32);
#pragma unroll
            for (int n = 0; n < NK; n++) {
                uint32_t b[4];
                ldsm4(b, ka + n * 8 * pitch + kp * 64);
                mma_bf16(s[n], a0, b[0], b[1]);
                mma_bf16(s2[n], a1, b[2], b[3]);
            }
        }
        const int p0 = begin + tile * LT_TOK;
        const bool edge = p0 + LT_TOK > pos0 + 1;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < NK; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                float v = (s[n][i] + s2[n][i]) * scale2;
                if (edge && p0 + key0 + n * 8 + 2 * tig + (i & 1) > pq[i >> 1]) v = -INFINITY;
                s[n][i] = v;
                mx[i >> 1] = fmaxf(mx[i >> 1], v);
            }
#pragma unroll
        for (int h = 0; h < 2; h++) {
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
            if (tig == 0) group_max[(mt * 16 + gid + 8 * h) * NG + kg] = mx[h];
        }
        __syncthreads();
        float alpha[MT][2], m_mine[2] = {0.f, 0.f};
        bool moved = false;
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int h = 0; h < 2; h++) {
                const float* g = group_max + (m * 16 + gid + 8 * h) * NG;
                float v = m_run[m][h];
#pragma unroll
                for (int k = 0; k < NG; k += 2) {
                    const float2 x = *reinterpret_cast<const float2*>(g + k);
                    v = fmaxf(v, fmaxf(x.x, x.y));
                }
                const float use = v == -INFINITY ? 0.f : v;
                alpha[m][h] = ex2(m_run[m][h] - use);
                moved |= m_run[m][h] != v;
                m_run[m][h] = v;
                if (m == mt) {
                    m_mine[h] = use;
                    l_run[h] *= alpha[m][h];
                }
            }
#pragma unroll
        for (int n = 0; n < NK; n++) {
            const float e0 = ex2(s[n][0] - m_mine[0]), e1 = ex2(s[n][1] - m_mine[0]), e2 = ex2(s[n][2] - m_mine[1]), e3 = ex2(s[n][3] - m_mine[1]);
            l_run[0] += e0 + e1, l_run[1] += e2 + e3;
            const int c = (key0 + n * 8 + 2 * tig) * 2;
            *reinterpret_cast<uint32_t*>(p_tile + (mt * 16 + gid) * LT_P_PITCH + c) = pack_bf16(e0, e1);
            *reinterpret_cast<uint32_t*>(p_tile + (mt * 16 + gid + 8) * LT_P_PITCH + c) = pack_bf16(e2, e3);
        }
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int n = 0; n < ND; n++) o[m][n][0] *= alpha[m][0], o[m][n][1] *= alpha[m][0], o[m][n][2] *= alpha[m][1], o[m][n][3] *= alpha[m][1];
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < LT_TOK / 16; kk++) {
            uint32_t pa[MT][4];
#pragma unroll
            for (int m = 0; m < MT; m++) ldsm4(pa[m], p_smem + (m * 16 + (lane & 15)) * LT_P_PITCH + kk * 32 + (lane >> 4) * 16);
            const uint32_t va = kt + (kk * 16 + (lane & 15)) * pitch + col0 * 2;
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
    cp_async_wait<0>();
    pdl_launch_dependents();
    // the key groups' sums meet
    __syncthreads();
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
        if (tig == 0) group_max[(mt * 16 + gid + 8 * h) * NG + kg] = l_run[h];
    }
    __syncthreads();
    const int64_t tile_id = (int64_t)blockIdx.z * gridDim.y + blockIdx.y;
    const int64_t share = (tile_id * n_splits + blockIdx.x) * QT;
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int qi = m * 16 + gid + 8 * h;
            if (qi >= n_queries) continue;
            float l = 0.f;
#pragma unroll
            for (int k = 0; k < NG; k++) l += group_max[qi * NG + k];
            const int head = head0 + qi % heads;
            if (n_splits == 1) {
                if (a.sink) l += ex2(a.sink[head] * 1.4426950408889634f - m_run[m][h]);
                const float f = 1.f / l;
                __nv_bfloat16* p = static_cast<__nv_bfloat16*>(a.out) + (int64_t)(row_first + qi / heads) * a.out_stride + (int64_t)head * DV + col0;
#pragma unroll
                for (int n = 0; n < ND; n++) *reinterpret_cast<uint32_t*>(p + n * 8 + 2 * tig) = pack_bf16(o[m][n][2 * h] * f, o[m][n][2 * h + 1] * f);
            } else {
                float* p = part_o + (share + qi) * DV + col0;
#pragma unroll
                for (int n = 0; n < ND; n++) *reinterpret_cast<float2*>(p + n * 8 + 2 * tig) = make_float2(o[m][n][2 * h], o[m][n][2 * h + 1]);
                if (warp == 0 && tig == 0) part_ml[share + qi] = make_float2(m_run[m][h], l);
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

template <int DV, int MT>
cudaError_t launch_one(tsb_ctx* ctx, cudaStream_t st, const LatentAttn& a, const WattnLaunch& l, int heads_per_tile, void* scratch) {
    const int head_tiles = (a.n_heads + heads_per_tile - 1) / heads_per_tile, base = l.n_tiles * head_tiles;
    const size_t smem = lt_smem<DV, MT>(a.keys.head_dim);
    const int per_sm = std::min(lt_per_sm(DV, MT), std::max(1, (int)(LT_SMEM_CAP / (smem + 1024))));
    const int splits = wattn_splits(ctx, 0, l, LT_TOK, 16 * MT, per_sm, base, std::min(wattn_part_queries(ctx), wattn_part_queries(ctx) * 256 / DV));
    const WattnScratch sc = wattn_scratch(ctx, scratch);
    static SmemOptIn configured;
    if (cudaError_t e = tsb_opt_in_smem(ctx, latent_attn_kernel<DV, MT>, LT_SMEM_CAP, configured); e != cudaSuccess) return e;
    cudaError_t e = tsb_launch(ctx, latent_attn_kernel<DV, MT>, dim3((unsigned)splits, (unsigned)head_tiles, (unsigned)l.n_tiles), dim3(LT_THREADS), smem, st,
                               true, a, l.tiles, l.tiles_per_group, l.rows_per_seq, l.rows_per_tile, heads_per_tile, sc.o, sc.ml, ctx->dev_error);
    if (e == cudaSuccess && splits > 1)
        e = tsb_launch(ctx, latent_merge_kernel, dim3(16 * MT, (unsigned)head_tiles, (unsigned)l.n_tiles), dim3(128), 0, st, true, a, l.tiles,
                       l.tiles_per_group, l.rows_per_seq, l.rows_per_tile, heads_per_tile, splits, 16 * MT, (const float*)sc.o, (const float2*)sc.ml);
    return e;
}
template <int DV>
cudaError_t launch_dim(tsb_ctx* ctx, cudaStream_t st, const LatentAttn& a, const WattnLaunch& l, const LatentTiling& t, void* scratch) {
    if (t.queries == 16) return launch_one<DV, 1>(ctx, st, a, l, t.heads, scratch);
    if (t.queries == 32) return launch_one<DV, 2>(ctx, st, a, l, t.heads, scratch);
    if constexpr (DV <= 256) return launch_one<DV, 4>(ctx, st, a, l, t.heads, scratch);
    return cudaErrorInvalidValue;
}

}  // namespace

bool latent_attn_dims(int kv_rank, int rot_dim, int* key_dim, int* value_dim) {
    for (int dv : {64, 128, 192, 256, 384, 512}) {
        if (kv_rank > dv) continue;
        const int dk = std::max((kv_rank + rot_dim + 31) / 32 * 32, dv);
        // the largest query tile of this width has to fit beside the ring
        const size_t smem = dv > 256 ? lt_smem<512, 2>(dk) : lt_smem<256, 4>(dk);
        if (smem > (size_t)LT_SMEM_CAP) return false;
        *key_dim = dk, *value_dim = dv;
        return true;
    }
    return false;
}

LatentTiling latent_attn_tiling(int n_heads, int value_dim, int most_rows) {
    const int most = value_dim > 256 ? 32 : 64;
    LatentTiling t;
    t.queries = 16;
    while (t.queries < most && t.queries < n_heads * most_rows) t.queries *= 2;
    const int head_tiles = (n_heads + t.queries - 1) / t.queries;
    t.heads = (n_heads + head_tiles - 1) / head_tiles;
    t.rows = std::max(1, std::min(most_rows, t.queries / t.heads));
    return t;
}

cudaError_t launch_latent_attn(tsb_ctx* ctx, cudaStream_t st, const LatentAttn& a, const AttnBatch& b, int most_rows, void* scratch) {
    const LatentTiling t = latent_attn_tiling(a.n_heads, a.value_dim, most_rows);
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
