// Matrix products with plain weights.  Three kernels:
//
//   plain_few_kernel   bfloat16, up to 16 token rows: bound by the weight stream.  A warp multiplies a tile of 16 (or
//                      2 x 16) weight rows on mma.sync.m16n8k16 with the tokens as the N side; the warps of a CTA split
//                      the columns and meet in shared memory.  The order of the columns inside a product is free as
//                      long as both operands agree, so a lane's fragments are contiguous 16-byte pieces of natural
//                      row-major rows: no repacking of weights or activations, no shared-memory staging.
//   plain_tc_kernel    bfloat16, more rows: tcgen05 tensor cores.  128 weight rows (M) x up to 256 tokens (N) per tile;
//                      a producer thread feeds 64-column slices of both operands through TMA into a ring of
//                      128-byte-swizzled stages, one thread issues the MMAs into one of two tensor-memory accumulators,
//                      eight warps run the epilogue of the tile before.  Persistent CTAs; products with too few tiles to
//                      fill the device are cut along K, the last run of a tile to finish adds the runs in order.
//   plain_f32_kernel   f32 throughout (fused multiply-adds on the CUDA cores): the reference-precision mode.
//
// All three share the epilogues: residual add, logits with a soft cap, and the projection epilogue that sends the rows of a
// packed matrix to buffers and straight into the paged cache, joins gate / up pairs and rotates the pairs of rotary parts.
#include <cuda.h>

#include <algorithm>
#include <cstdlib>
#include <map>
#include <mutex>

#include "gemm_plain.cuh"
#include "tc05.cuh"

namespace {

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// act(z) in f32.  0.5 z (1 + tanh(u)) = z / (1 + exp(-2u)); the reduced-precision path takes the fast exponential and
// division (relative error a few 2^-22), the f32 path the library's.
template <typename T>
__device__ __forceinline__ float activate(int act, float z) {
    if (act == PLAIN_RELU2) return fmaxf(z, 0.f) * fmaxf(z, 0.f);
    const float u = act == PLAIN_GELU_TANH ? 1.5957691216057308f * (z + 0.044715f * z * z * z) : z;  // 2 sqrt(2 / pi)
    if (sizeof(T) == 4) {
        if (act == PLAIN_GELU_TANH) return 0.5f * z * (1.f + tanhf(0.5f * u));
        return z / (1.f + expf(-u));
    }
    return __fdividef(z, 1.f + __expf(-u));
}

__device__ __forceinline__ float get(const float* p) { return *p; }
__device__ __forceinline__ float get(const __nv_bfloat16* p) { return __bfloat162float(*p); }

// Where row n of the matrix goes (PLAIN_MIXER).
struct SegAt {
    int kind = -1, col = 0, gate_col = 0;  // -1: nowhere
    void* p = nullptr;
    int64_t stride = 0;
    const void* gate = nullptr;
    int64_t gate_stride = 0;
    int act = -1;
};
__device__ __forceinline__ SegAt seg_at(const PlainEpi& e, int n) {
    SegAt at;
    int first = 0;
#pragma unroll
    for (int k = 0; k < PLAIN_SEGS; k++) {
        if (k >= e.n_seg) break;
        const PlainSeg& s = e.seg[k];
        if (n < s.end) {
            const int g = (n - first) / s.per, i = (n - first) - g * s.per;
            if (i < s.valid) {
                at.kind = s.kind, at.col = g * s.step + i, at.p = s.p, at.stride = s.stride;
                at.gate = s.gate, at.gate_stride = s.gate_stride, at.gate_col = g * s.gate_step + i, at.act = s.act;
            }
            break;
        }
        first = s.end;
    }
    return at;
}
template <typename T>
__device__ __forceinline__ void seg_put(const PlainEpi& e, const SegAt& at, int t, float v, uint32_t* err) {
    if (at.kind == PLAIN_SEG_TYPED) {
        if (at.act >= 0) v = activate<T>(at.act, v);
        if (at.gate) {
            const float z = get(static_cast<const T*>(at.gate) + (int64_t)t * at.gate_stride + at.gate_col);
            v *= 1.f / (1.f + expf(-z));
        }
        put(static_cast<T*>(at.p) + (int64_t)t * at.stride + at.col, v);
    } else if (at.kind == PLAIN_SEG_F32) {
        static_cast<float*>(at.p)[(int64_t)t * at.stride + at.col] = v;
    } else if (at.kind == PLAIN_SEG_CACHE) {
        const tsb_row_desc& rd = e.rows[t];
        T* p = key_row<T>(e.keys, rd.seq, rd.base + rd.slot);
        if (p) put(p + at.stride + at.col, v);
        else atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
    }
}

template <typename T>
__device__ __forceinline__ void epi_one(const PlainEpi& e, int t, int n, float v, uint32_t* err) {
    if (e.kind == PLAIN_STORE) {
        if (n < e.n_valid) e.y[(int64_t)t * e.y_stride + n] = e.cap > 0.f ? e.cap * tanhf(v / e.cap) : v;
    } else if (e.kind == PLAIN_ADD) {
        if (n < e.n_valid) {
            float* y = e.y + (int64_t)t * e.y_stride + n;
            *y = fmaf(e.alpha, *y, e.beta * v);
        }
    } else {
        if (e.bias) v += e.bias[n];
        seg_put<T>(e, seg_at(e, n), t, v, err);
    }
}
template <typename T>
__device__ __forceinline__ void epi_pair(const PlainEpi& e, int t, int pair, float g, float u, uint32_t* err) {
    if (pair >= e.n_pairs) return;
    const PlainRotate& r = e.rot;
    if (r.half == 0) {
        put(static_cast<T*>(e.a) + (int64_t)t * e.a_stride + pair, activate<T>(e.act, g) * u);
        return;
    }
    const int head = pair / r.half, i = pair - head * r.half;
    const float2 cs = r.table[(int64_t)t * r.half + i];
    const float lo = fmaf(g, cs.x, -u * cs.y), hi = fmaf(u, cs.x, g * cs.y);
    if (head < r.n_heads) {
#pragma unroll
        for (int k = 0; k < 2; k++) {
            if (!r.q[k]) continue;
            T* p = static_cast<T*>(r.q[k]) + (int64_t)t * r.q_stride[k] + head * r.q_step[k] + r.q_off[k] + i;
            put(p, lo), put(p + r.half, hi);
        }
    } else {
        const tsb_row_desc& rd = e.rows[t];
        T* p = key_row<T>(e.keys, rd.seq, rd.base + rd.slot);
        if (p) put(p + r.key_off + i, lo), put(p + r.key_off + r.half + i, hi);
        else atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
    }
}

// does any output come from the rows at and after row0 (up to the next segment, or to the end of the group)?
__device__ __forceinline__ bool tile_used(const PlainEpi& e, int row0, int group_rows) {
    if (row0 >= e.pair_row0) return (row0 - e.pair_row0) / 2 < e.n_pairs;
    if (e.kind != PLAIN_MIXER) return row0 < e.n_valid;
    return e.n_seg > 0 && row0 < e.seg[e.n_seg - 1].end && (group_rows == 0 || row0 % group_rows < e.seg[0].valid);
}

// ------------------------------------------------------------------ few rows
constexpr int FEW_WARPS = 8;
constexpr int FEW_UNROLL = 4;  // 64-column units in flight per warp

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint4 ldg_stream(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// NT token tiles of eight, MT row tiles of sixteen.  WK warps split the columns of a row tile; products with few columns have
// several row tiles per CTA instead.  blockIdx.y: which 8 NT tokens; EXPERTS: which chunk of slots.
template <int NT, int MT, int WK, bool EXPERTS>
__global__ void __launch_bounds__(FEW_WARPS * 32, 2)
    plain_few_kernel(const __nv_bfloat16* __restrict__ w, int cols, int group_rows, int group_cols, const __nv_bfloat16* x, const __nv_bfloat16* x2,
                     int64_t x_stride, int tokens, const __grid_constant__ PlainEpi epi, const __grid_constant__ PlainExperts ex, uint32_t* __restrict__ err) {
    constexpr int U = MT == 1 ? FEW_UNROLL : FEW_UNROLL / 2;
    constexpr int TOK = NT * 8, WROWS = MT * 16, ROWS = WROWS * (FEW_WARPS / WK);
    __shared__ float red[FEW_WARPS][WROWS][TOK + 1];
    const int warp = (threadIdx.x >> 5) % WK, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    const int wrow = (threadIdx.x >> 5) / WK * WROWS, row0 = blockIdx.x * ROWS;
    int tok0 = blockIdx.y * TOK;
    if (EXPERTS) {  // which rows of which matrix is known only now
        pdl_wait();
        if ((int)blockIdx.y >= *ex.n_chunks) return;
        const ExpertChunk c = ex.chunks[blockIdx.y];
        w += (int64_t)c.expert * gridDim.x * ROWS * cols;
        tok0 = c.first, tokens = min(c.n, TOK);
    } else {
        tokens = min(tokens - tok0, TOK);
    }
    const int units = cols / 64;
    const bool pairs = row0 >= epi.pair_row0;
    if (!tile_used(epi, row0, group_rows)) return;  // padding between the mixer's rows and the pairs, or behind a group
    const __nv_bfloat16* wp = w + (int64_t)(row0 + wrow + g) * cols + 8 * t4;
    // a unit of 64 columns is two k = 32 halves; per half the lane holds columns 8 t4 .. 8 t4 + 7 of its two rows
    uint4 wa[U][MT][4];
    auto load_w = [&](int i, int u) {
#pragma unroll
        for (int m = 0; m < MT; m++) {
            const __nv_bfloat16* p = wp + (int64_t)m * 16 * cols + (int64_t)u * 64;
            wa[i][m][0] = ldg_stream(p);
            wa[i][m][1] = ldg_stream(p + (int64_t)8 * cols);
            wa[i][m][2] = ldg_stream(p + 32);
            wa[i][m][3] = ldg_stream(p + (int64_t)8 * cols + 32);
        }
    };
#pragma unroll
    for (int i = 0; i < U; i++)
        if (warp + i * WK < units) load_w(i, warp + i * WK);  // weights do not depend on the preceding kernel
    if (!EXPERTS) pdl_wait();
    const __nv_bfloat16* xb = (pairs ? x2 : x) + 8 * t4 + (group_rows ? row0 / group_rows * group_cols : 0);
    int64_t x_at[NT];
#pragma unroll
    for (int n = 0; n < NT; n++) {
        const int t = tok0 + n * 8 + g;
        x_at[n] = (EXPERTS && ex.token_of ? (n * 8 + g < tokens ? ex.token_of[t] : 0) : t) * x_stride;
    }
    float acc[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int n = 0; n < NT; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) acc[m][n][i] = 0.f;
    for (int u0 = warp; u0 < units; u0 += U * WK) {
#pragma unroll
        for (int i = 0; i < U; i++) {
            const int u = u0 + i * WK;
            if (u >= units) break;
#pragma unroll
            for (int n = 0; n < NT; n++) {
                const __nv_bfloat16* xp = xb + x_at[n] + (int64_t)u * 64;
                uint4 b0 = make_uint4(0, 0, 0, 0), b1 = b0;
                if (n * 8 + g < tokens) b0 = *reinterpret_cast<const uint4*>(xp), b1 = *reinterpret_cast<const uint4*>(xp + 32);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    const uint32_t a0[4] = {wa[i][m][0].x, wa[i][m][1].x, wa[i][m][0].y, wa[i][m][1].y};
                    const uint32_t a1[4] = {wa[i][m][0].z, wa[i][m][1].z, wa[i][m][0].w, wa[i][m][1].w};
                    const uint32_t a2[4] = {wa[i][m][2].x, wa[i][m][3].x, wa[i][m][2].y, wa[i][m][3].y};
                    const uint32_t a3[4] = {wa[i][m][2].z, wa[i][m][3].z, wa[i][m][2].w, wa[i][m][3].w};
                    mma_bf16(acc[m][n], a0, b0.x, b0.y);
                    mma_bf16(acc[m][n], a1, b0.z, b0.w);
                    mma_bf16(acc[m][n], a2, b1.x, b1.y);
                    mma_bf16(acc[m][n], a3, b1.z, b1.w);
                }
            }
            const int un = u + U * WK;
            if (un < units) load_w(i, un);
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int n = 0; n < NT; n++) {
            float(*mine)[TOK + 1] = red[threadIdx.x >> 5];
            mine[m * 16 + g][n * 8 + 2 * t4] = acc[m][n][0];
            mine[m * 16 + g][n * 8 + 2 * t4 + 1] = acc[m][n][1];
            mine[m * 16 + g + 8][n * 8 + 2 * t4] = acc[m][n][2];
            mine[m * 16 + g + 8][n * 8 + 2 * t4 + 1] = acc[m][n][3];
        }
    __syncthreads();
    auto total = [&](int r, int t) {
        float v = 0.f;
#pragma unroll
        for (int i = 0; i < WK; i++) v += red[r / WROWS * WK + i][r % WROWS][t];
        return v;
    };
    if (pairs) {
        for (int i = threadIdx.x; i < ROWS / 2 * tokens; i += FEW_WARPS * 32) {
            const int p = i % (ROWS / 2), t = i / (ROWS / 2);
            const int r = (p >> 3) * 16 + (p & 7);
            epi_pair<__nv_bfloat16>(epi, tok0 + t, (row0 - epi.pair_row0) / 2 + p, total(r, t), total(r + 8, t), err);
        }
    } else {
        for (int i = threadIdx.x; i < ROWS * tokens; i += FEW_WARPS * 32) {
            const int r = i % ROWS, t = i / ROWS;
            epi_one<__nv_bfloat16>(epi, tok0 + t, row0 + r, total(r, t), err);
        }
    }
}

// ------------------------------------------------------------------ f32
constexpr int F32_TILE = 64, F32_K = 16;
// 256 threads, 64 rows x 64 tokens, 4 x 4 per thread.  A thread's four rows are {0, 8, 16, 24} + r within a 32-row half:
// both halves of a gate / up pair are its own.
template <bool EXPERTS>
__global__ void __launch_bounds__(256)
    plain_f32_kernel(const float* __restrict__ w, int cols, int group_rows, int group_cols, const float* x, const float* x2, int64_t x_stride, int tokens,
                     const __grid_constant__ PlainEpi epi, const __grid_constant__ PlainExperts ex, uint32_t* __restrict__ err) {
    __shared__ float ws[F32_K][F32_TILE + 4], xs[F32_K][F32_TILE + 4];
    const int row0 = blockIdx.x * F32_TILE;
    int tok0 = blockIdx.y * F32_TILE;
    const bool pairs = row0 >= epi.pair_row0;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const int rbase = (ty >> 3) * 32 + (ty & 7);
    pdl_wait();
    if (EXPERTS) {
        if ((int)blockIdx.y >= *ex.n_chunks) return;
        const ExpertChunk c = ex.chunks[blockIdx.y];
        w += (int64_t)c.expert * gridDim.x * F32_TILE * cols;
        tok0 = c.first, tokens = c.first + min(c.n, F32_TILE);
    }
    const float* xb = (pairs ? x2 : x) + (group_rows ? row0 / group_rows * group_cols : 0);
    float acc[4][4] = {};
    const int lr = threadIdx.x >> 2, lc = (threadIdx.x & 3) * 4;
    const int64_t x_at = (EXPERTS && ex.token_of ? (tok0 + lr < tokens ? ex.token_of[tok0 + lr] : 0) : tok0 + lr) * x_stride;
    for (int k0 = 0; k0 < cols; k0 += F32_K) {
        const float4 a = *reinterpret_cast<const float4*>(w + (int64_t)(row0 + lr) * cols + k0 + lc);
        float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
        if (tok0 + lr < tokens) b = *reinterpret_cast<const float4*>(xb + x_at + k0 + lc);
        ws[lc][lr] = a.x, ws[lc + 1][lr] = a.y, ws[lc + 2][lr] = a.z, ws[lc + 3][lr] = a.w;
        xs[lc][lr] = b.x, xs[lc + 1][lr] = b.y, xs[lc + 2][lr] = b.z, xs[lc + 3][lr] = b.w;
        __syncthreads();
        float part[4][4] = {};  // sums of a slice first: rounding grows with the number of slices, not of columns
#pragma unroll
        for (int k = 0; k < F32_K; k++) {
            float wv[4], xv[4];
#pragma unroll
            for (int i = 0; i < 4; i++) wv[i] = ws[k][rbase + 8 * i], xv[i] = xs[k][tx + 16 * i];
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) part[i][j] = fmaf(wv[i], xv[j], part[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) acc[i][j] += part[i][j];
        __syncthreads();
    }
    pdl_launch_dependents();
#pragma unroll
    for (int j = 0; j < 4; j++) {
        const int t = tok0 + tx + 16 * j;
        if (t >= tokens) continue;
        if (pairs) {
#pragma unroll
            for (int h = 0; h < 2; h++) {
                const int r = row0 - epi.pair_row0 + (ty >> 3) * 32 + 16 * h;  // the pair group's first row
                epi_pair<float>(epi, t, r / 2 + (ty & 7), acc[2 * h][j], acc[2 * h + 1][j], err);
            }
        } else {
#pragma unroll
            for (int i = 0; i < 4; i++) epi_one<float>(epi, t, row0 + rbase + 8 * i, acc[i][j], err);
        }
    }
}

// ------------------------------------------------------------------ tensor memory
constexpr int TCG_M = 128;        // weight rows per tile
constexpr int TCG_K = 64;         // columns per stage (128 bytes: one swizzle row)
constexpr int TCG_NMAX = 256;     // tokens per tile
constexpr int TCG_EPI_WARPS = 8;  // warp w owns tensor-memory lanes 32 (w % 4) .. + 31 and every other run of sixteen tokens
constexpr int TCG_THREADS = (TCG_EPI_WARPS + 2) * 32;
constexpr int TCG_HEADER = 1024;
constexpr int TCG_MAX_STAGES = 8;
constexpr int TCG_SMEM_CAP = 224 * 1024;
constexpr int TCG_TICKETS = 4096;
constexpr int TCG_MAX_SPLITS = 16;

struct TcgBars {
    uint64_t full[TCG_MAX_STAGES], empty[TCG_MAX_STAGES];
    uint64_t acc_full[2], acc_empty[2];
    uint32_t tmem_base, failed, ticket;
};

__device__ __forceinline__ void tcg_g2s_2d(uint32_t dst_smem, const CUtensorMap* map, int x, int y, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst_smem),
                 "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(smem_u32(bar))
                 : "memory");
}

// Where the outputs of one thread of the tensor-memory epilogue go: row n of the matrix, or, in a tile of pairs, every other token of
// the pair that the row belongs to.
struct TcgOut {
    SegAt at;             // rows with a destination of their own
    bool pairs = false, cache = false, in = false;
    float bias = 0.f;
    int tok0, pair = 0, head = 0, col = 0;  // head, col: of a rotated pair
    __device__ __forceinline__ TcgOut(const PlainEpi& e, int row0, int n, int lane, int tok0_) : tok0(tok0_) {
        pairs = row0 >= e.pair_row0;
        if (e.kind != PLAIN_MIXER) {
            in = n < e.n_valid, at.col = n;
        } else if (!pairs) {
            at = seg_at(e, n);
            in = at.kind >= 0, cache = at.kind == PLAIN_SEG_CACHE;
            if (e.bias && in) bias = e.bias[n];
        } else {
            pair = ((n & ~31) - e.pair_row0) / 2 + (lane >> 4) * 8 + (lane & 7);
            in = pair < e.n_pairs;
            if (e.rot.half > 0) head = pair / e.rot.half, col = pair - head * e.rot.half, cache = in && head >= e.rot.n_heads;
        }
    }
    static __device__ __forceinline__ float gate_of(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

    // sixteen tokens from tok0 + c0 on
    template <int KIND>
    __device__ __forceinline__ void store(const PlainEpi& e, float (&v)[16], int c0, int n_tok, int lane, bool to_cache, uint32_t* err) const {
        const int t0 = tok0 + c0, left = in ? n_tok - c0 : 0;  // tokens this thread stores
        if (KIND != PLAIN_MIXER) {
            float* y = e.y + (int64_t)t0 * e.y_stride + (in ? at.col : 0);
            const int64_t step = e.y_stride;
            if (KIND == PLAIN_ADD) {
                float old[16];
#pragma unroll
                for (int j = 0; j < 16; j++) old[j] = j < left ? y[j * step] : 0.f;
#pragma unroll
                for (int j = 0; j < 16; j++)
                    if (j < left) y[j * step] = fmaf(e.alpha, old[j], e.beta * v[j]);
            } else {
                if (e.cap > 0.f) {
#pragma unroll 1
                    for (int k = 0; k < 16; k++) {  // rotates the array through one element: one copy of the function
                        const float x = e.cap * tanhf(v[0] / e.cap);
#pragma unroll
                        for (int j = 0; j < 15; j++) v[j] = v[j + 1];
                        v[15] = x;
                    }
                }
#pragma unroll
                for (int j = 0; j < 16; j++)
                    if (j < left) y[j * step] = v[j];
            }
        } else if (!pairs) {
            if (e.bias) {
#pragma unroll
                for (int j = 0; j < 16; j++) v[j] += bias;
            }
            if (at.kind == PLAIN_SEG_F32) {
                float* y = static_cast<float*>(at.p) + (int64_t)t0 * at.stride + at.col;
#pragma unroll
                for (int j = 0; j < 16; j++)
                    if (j < left) y[j * at.stride] = v[j];
            } else if (at.kind == PLAIN_SEG_TYPED) {
                if (at.act >= 0) {
#pragma unroll
                    for (int j = 0; j < 16; j++) v[j] = activate<__nv_bfloat16>(at.act, v[j]);
                }
                if (at.gate) {
                    const __nv_bfloat16* g = static_cast<const __nv_bfloat16*>(at.gate) + (int64_t)t0 * at.gate_stride + at.gate_col;
                    float z[16];
#pragma unroll
                    for (int j = 0; j < 16; j++) z[j] = j < left ? __bfloat162float(g[j * at.gate_stride]) : 0.f;
#pragma unroll
                    for (int j = 0; j < 16; j++) v[j] *= gate_of(z[j]);
                }
                __nv_bfloat16* y = static_cast<__nv_bfloat16*>(at.p) + (int64_t)t0 * at.stride + at.col;
#pragma unroll
                for (int j = 0; j < 16; j++)
                    if (j < left) put(y + j * at.stride, v[j]);
            }
            if (to_cache) {  // the lanes look up the sixteen tokens' rows, every lane stores to all of them
                const __nv_bfloat16* row = cache_row(e, t0, n_tok - c0, lane, err);
#pragma unroll
                for (int j = 0; j < 16; j++) {
                    __nv_bfloat16* p = reinterpret_cast<__nv_bfloat16*>(__shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(row), j));
                    if (cache && p) put(p + at.stride + at.col, v[j]);
                }
            }
        } else {
            // The two rows of a pair sit eight lanes apart: after one exchange the lower lane has both coordinates of the even token, the
            // upper lane those of the odd one.
            const bool upper = lane & 8;
            const __nv_bfloat16* row = to_cache ? cache_row(e, t0, n_tok - c0, lane, err) : nullptr;
            const PlainRotate& r = e.rot;
#pragma unroll
            for (int j = 0; j < 16; j += 2) {
                const float other = __shfl_xor_sync(0xffffffffu, upper ? v[j] : v[j + 1], 8);
                const float a = upper ? other : v[j], b = upper ? v[j + 1] : other;
                const int k = j + (upper ? 1 : 0);
                __nv_bfloat16* p = nullptr;
                if (to_cache) p = reinterpret_cast<__nv_bfloat16*>(__shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(row), k));
                if (k >= left) continue;
                if (r.half == 0) {
                    put(static_cast<__nv_bfloat16*>(e.a) + (int64_t)(t0 + k) * e.a_stride + pair, activate<__nv_bfloat16>(e.act, a) * b);
                    continue;
                }
                const float2 cs = r.table[(int64_t)(t0 + k) * r.half + col];
                const float lo = fmaf(a, cs.x, -b * cs.y), hi = fmaf(b, cs.x, a * cs.y);
                if (cache) {
                    if (p) put(p + r.key_off + col, lo), put(p + r.key_off + r.half + col, hi);
                } else {
#pragma unroll
                    for (int x = 0; x < 2; x++) {
                        if (!r.q[x]) continue;
                        __nv_bfloat16* q = static_cast<__nv_bfloat16*>(r.q[x]) + (int64_t)(t0 + k) * r.q_stride[x] + head * r.q_step[x] + r.q_off[x] + col;
                        put(q, lo), put(q + r.half, hi);
                    }
                }
            }
        }
    }

private:
    static __device__ __forceinline__ __nv_bfloat16* cache_row(const PlainEpi& e, int t0, int left, int lane, uint32_t* err) {
        if ((lane & 15) >= left) return nullptr;
        const tsb_row_desc& rd = e.rows[t0 + (lane & 15)];
        __nv_bfloat16* p = key_row<__nv_bfloat16>(e.keys, rd.seq, rd.base + rd.slot);
        if (!p) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        return p;
    }
};

// Work item i: token tile i % n_tok_tiles, then the K run, then the row tile - neighbouring CTAs share weight rows.  EXPERTS: expert by
// expert, with as many token tiles as its slots need; the counts are on the device.
constexpr int TCG_EXPERT_BYTES = 2 * (EXPERTS_MAX + 2) * sizeof(int);  // behind the ring: first slots, first token tiles
template <int KIND, bool EXPERTS>
__global__ void __launch_bounds__(TCG_THREADS, 1)
    plain_tc_kernel(const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap xmap, const __grid_constant__ CUtensorMap x2map,
                    int n_row_tiles, int n_tok_tiles, int units, int ksplit, int nt, int stages, int tokens, int group_rows, int group_cols,
                    const __grid_constant__ PlainEpi epi, const __grid_constant__ PlainExperts ex, float* __restrict__ part, uint32_t* __restrict__ tickets,
                    uint32_t* __restrict__ err) {
    extern __shared__ __align__(1024) uint8_t smem[];
    TcgBars* bars = reinterpret_cast<TcgBars*>(smem);
    uint8_t* ring = smem + TCG_HEADER;
    const int stage_bytes = (TCG_M + nt) * 128;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int n_items = n_row_tiles * n_tok_tiles * ksplit;
    int *slot0 = reinterpret_cast<int*>(ring + stages * stage_bytes), *tile0 = slot0 + EXPERTS_MAX + 2;
    const int run_units = (units + ksplit - 1) / ksplit;
    const uint32_t tmem_cols = nt <= 16 ? 32u : nt <= 32 ? 64u : nt <= 64 ? 128u : nt <= 128 ? 256u : 512u;
    if (threadIdx.x == 0) {
        for (int i = 0; i < stages; i++) mbar_init(&bars->full[i], 1), mbar_init(&bars->empty[i], 1);
        for (int i = 0; i < 2; i++) mbar_init(&bars->acc_full[i], 1), mbar_init(&bars->acc_empty[i], TCG_EPI_WARPS);
        bars->failed = 0;
        mbar_fence_init();
    }
    if (warp == TCG_EPI_WARPS + 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&bars->tmem_base)), "r"(tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    if (EXPERTS) {
        pdl_wait();  // the lists come from the kernels before
        for (int e = threadIdx.x; e <= ex.n; e += TCG_THREADS) slot0[e] = ex.first[e];
        __syncthreads();
        if (warp == 0) {
            int sum = 0;
            for (int e0 = 0; e0 < ex.n; e0 += 32) {
                const int e = e0 + lane, n = e < ex.n ? (slot0[e + 1] - slot0[e] + nt - 1) / nt : 0;
                int s = n;
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const int v = __shfl_up_sync(0xffffffffu, s, o);
                    if (lane >= o) s += v;
                }
                if (e < ex.n) tile0[e] = sum + s - n;
                sum += __shfl_sync(0xffffffffu, s, 31);
            }
            if (lane == 0) tile0[ex.n] = sum;
        }
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bars->tmem_base;
    if (EXPERTS) n_items = tile0[ex.n] * n_row_tiles;
    struct Item {
        int tok, run, row, u0, n, tok0, n_tok, wrow;  // wrow: row of the matrix behind the weight map
    };
    auto item_of = [&](int i) {
        Item it;
        if (EXPERTS) {
            int lo = 0, hi = ex.n;  // the last expert that starts at or before item i, empty ones skipped by the search's upper end
            while (hi - lo > 1) {
                const int mid = (lo + hi) >> 1;
                if (tile0[mid] * n_row_tiles <= i) lo = mid;
                else hi = mid;
            }
            const int tiles = tile0[lo + 1] - tile0[lo], j = i - tile0[lo] * n_row_tiles;
            it.tok = j % tiles, it.row = j / tiles, it.run = 0, it.u0 = 0, it.n = units;
            // the expert's slots over its tiles, evenly
            const int n = slot0[lo + 1] - slot0[lo], width = ((n + tiles - 1) / tiles + 15) & ~15;
            it.tok0 = slot0[lo] + min(n, it.tok * width), it.n_tok = min(width, slot0[lo + 1] - it.tok0);
            it.wrow = (lo * n_row_tiles + it.row) * TCG_M;
            return it;
        }
        it.tok = i % n_tok_tiles;
        it.run = (i / n_tok_tiles) % ksplit;
        it.row = i / n_tok_tiles / ksplit;
        it.u0 = it.run * run_units;
        it.n = min(units, it.u0 + run_units) - it.u0;
        it.tok0 = it.tok * nt, it.n_tok = min(nt, tokens - it.tok0), it.wrow = it.row * TCG_M;
        return it;
    };

    if (warp == TCG_EPI_WARPS) {
        if (lane == 0) {
            // ---- producer.  Weights do not depend on the preceding kernel, activations do: the first stages' weight
            // slices start before the wait, their activation slices after it.
            bool ok = true;
            uint32_t it = 0;
            int early = 0;  // stages whose weight slice was fetched ahead
            const bool has_work = (int)blockIdx.x < n_items;
            if (has_work && !EXPERTS) {
                const Item w0 = item_of(blockIdx.x);
                early = min(stages, w0.n);
                for (int s = 0; s < early; s++) {
                    mbar_expect_tx(&bars->full[s], (uint32_t)stage_bytes);
                    tcg_g2s_2d(smem_u32(ring + s * stage_bytes), &wmap, (w0.u0 + s) * TCG_K, w0.wrow, &bars->full[s]);
                }
            }
            if (!EXPERTS) pdl_wait();
            for (int i = blockIdx.x; i < n_items && ok; i += gridDim.x) {
                const Item w = item_of(i);
                const CUtensorMap* xm = w.row * TCG_M >= epi.pair_row0 ? &x2map : &xmap;
                const int x_col0 = group_rows ? w.row * TCG_M / group_rows * group_cols : 0;  // a multiple of the stage's 64 columns
                for (int u = 0; u < w.n && ok; u++, it++) {
                    const int s = it % stages;
                    const uint32_t dst = smem_u32(ring + s * stage_bytes);
                    if ((int)it >= early) {
                        if ((int)it >= stages) ok = mbar_wait(&bars->empty[s], ((it / stages) - 1) & 1, err);
                        if (!ok) break;
                        mbar_expect_tx(&bars->full[s], (uint32_t)stage_bytes);
                        tcg_g2s_2d(dst, &wmap, (w.u0 + u) * TCG_K, w.wrow, &bars->full[s]);
                    }
                    tcg_g2s_2d(dst + TCG_M * 128, xm, x_col0 + (w.u0 + u) * TCG_K, w.tok0, &bars->full[s]);
                }
            }
            if (!ok) bars->failed = 1;
            // no copy is in flight when the CTA leaves, also when another role has given up
            for (uint32_t k = it > (uint32_t)stages ? it - stages : 0; k < it; k++) mbar_wait(&bars->full[k % stages], (k / stages) & 1, err);
        }
    } else if (warp == TCG_EPI_WARPS + 1) {
        // ---- MMA issue: the warp walks the items together, lane 0 issues.  f32 accumulate, bfloat16 operands, both
        // K-major and 128-byte swizzled (eight-row groups 1024 bytes apart; a K = 16 step moves the start by 32 bytes)
        const uint32_t leader = lane == 0 ? 1u : 0u;
        auto idesc_of = [](int n) { return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(TCG_M >> 4) << 24); };
        constexpr uint64_t DESC = ((uint64_t)1u << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) | (2ull << 61);
        bool ok = true;
        uint32_t it = 0, tile = 0;
        for (int i = blockIdx.x; i < n_items && ok; i += gridDim.x, tile++) {
            const Item w = item_of(i);
            const uint32_t buf = tile & 1;
            if (tile >= 2) ok = __all_sync(0xffffffffu, mbar_wait(&bars->acc_empty[buf], ((tile >> 1) - 1) & 1, err));
            if (!ok) break;
            tc_fence_after();
            const uint32_t d = tmem + buf * (uint32_t)nt;
            // an expert's tile multiplies only the tokens it has
            const uint32_t idesc = EXPERTS ? idesc_of(max(16, (w.n_tok + 15) & ~15)) : idesc_of(nt);
            for (int u = 0; u < w.n; u++, it++) {
                const int s = it % stages;
                ok = __all_sync(0xffffffffu, mbar_wait(&bars->full[s], (it / stages) & 1, err));
                if (!ok) break;
                tc_fence_after();
                const uint32_t a_addr = smem_u32(ring + s * stage_bytes);
                const uint64_t da = DESC | (uint64_t)((a_addr >> 4) & 0x3FFFu);
                const uint64_t db = DESC | (uint64_t)(((a_addr + TCG_M * 128) >> 4) & 0x3FFFu);
                if (u == 0) tc_mma_ss<false>(leader, d, da, db, idesc);
                else tc_mma_ss<true>(leader, d, da, db, idesc);
#pragma unroll
                for (int ks = 1; ks < TCG_K / 16; ks++) tc_mma_ss<true>(leader, d, da + 2u * ks, db + 2u * ks, idesc);
                tc_commit_if(leader, &bars->empty[s]);
            }
            if (ok) tc_commit_if(leader, &bars->acc_full[buf]);
        }
        if (!ok && lane == 0) bars->failed = 1;
    } else {
        // ---- epilogue: two threads per weight row of the tile, columns = tokens.  One destination per tile and thread, one short
        // loop per kind of destination: the code of a kind has to stay in the instruction cache.
        if (!EXPERTS) pdl_wait();  // the residual stream and the cache belong to earlier kernels too
        bool ok = true;
        uint32_t tile = 0;
        const int quad = warp & 3, first16 = (warp >> 2) * 16;
        const uint32_t lane_base = (uint32_t)(quad * 32) << 16;
        for (int i = blockIdx.x; i < n_items; i += gridDim.x, tile++) {
            const Item w = item_of(i);
            const uint32_t buf = tile & 1;
            if (ok) ok = mbar_wait(&bars->acc_full[buf], (tile >> 1) & 1, err);
            tc_fence_after();
            const uint32_t src = tmem + lane_base + buf * (uint32_t)nt;
            const int n = w.row * TCG_M + quad * 32 + lane;
            const int tok0 = w.tok0, n_tok = w.n_tok;
            bool finish = ok;
            const float* all = nullptr;
            if (ksplit > 1) {
                // a run of a cut tile: leave the sums, take a ticket; whoever takes the last one adds the runs in order
                const int tix = w.row * n_tok_tiles + w.tok;
                float* mine = part + ((int64_t)tix * ksplit + w.run) * (TCG_M * nt) + quad * 32 + lane;
                for (int c0 = first16; c0 < n_tok; c0 += 32) {
                    uint32_t r[16];
                    tc_ld16(src + c0, r);
                    tc_wait_ld();
#pragma unroll
                    for (int j = 0; j < 16; j++) mine[(c0 + j) * TCG_M] = ok ? __uint_as_float(r[j]) : 0.f;
                }
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(&bars->acc_empty[buf]);
                __threadfence();
                asm volatile("bar.sync 1, %0;" ::"n"(TCG_EPI_WARPS * 32) : "memory");
                if (threadIdx.x == 0) {
                    const uint32_t t = atomicAdd(&tickets[tix], 1u);
                    if (t == (uint32_t)ksplit - 1) tickets[tix] = 0;
                    bars->ticket = t;
                }
                asm volatile("bar.sync 1, %0;" ::"n"(TCG_EPI_WARPS * 32) : "memory");
                finish = bars->ticket == (uint32_t)ksplit - 1;
                __threadfence();
                all = part + (int64_t)tix * ksplit * (TCG_M * nt) + quad * 32 + lane;
                asm volatile("bar.sync 1, %0;" ::"n"(TCG_EPI_WARPS * 32) : "memory");  // the ticket word is reused by the next tile
            }
            const TcgOut out(epi, w.row * TCG_M, n, lane, tok0);
            const bool to_cache = KIND == PLAIN_MIXER && __any_sync(0xffffffffu, out.cache);
            // one loop over the tile's tokens, sixteen at a time
            if (finish)
                for (int c0 = first16; c0 < n_tok; c0 += 32) {
                    float v[16];
                    __syncwarp();
                    if (ksplit == 1) {
                        uint32_t r[16];
                        tc_ld16(src + c0, r);
                        tc_wait_ld();
#pragma unroll
                        for (int j = 0; j < 16; j++) v[j] = __uint_as_float(r[j]);
                    } else {
#pragma unroll
                        for (int j = 0; j < 16; j++) v[j] = 0.f;
                        for (int k = 0; k < ksplit; k++) {
#pragma unroll
                            for (int j = 0; j < 16; j++) v[j] += __ldcg(all + (int64_t)k * (TCG_M * nt) + (c0 + j) * TCG_M);
                        }
                    }
                    out.store<KIND>(epi, v, c0, n_tok, lane, to_cache, err);
                }
            if (ksplit == 1) {
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(&bars->acc_empty[buf]);
            }
        }
        if (!ok && lane == 0) bars->failed = 1;
    }
    pdl_launch_dependents();
    tc_fence_before();
    __syncthreads();
    if (warp == TCG_EPI_WARPS + 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(tmem_cols) : "memory");
    }
}

// 2-D bfloat16 tensor map over [rows][cols], box 64 columns x box_rows rows, 128-byte swizzle.  Encoding goes through the
// driver entry point (no link against libcuda); maps are kept per (address, shape).
cudaError_t tcg_map(const void* p, int64_t rows, int64_t cols, int64_t stride, int box_rows, CUtensorMap* out) {
    typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                 const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
    static std::mutex mu;
    static EncodeFn encode = nullptr;
    struct Key {
        const void* p;
        int64_t rows, cols, stride;
        int box;
        bool operator<(const Key& o) const {
            return p != o.p ? p < o.p : rows != o.rows ? rows < o.rows : cols != o.cols ? cols < o.cols : stride != o.stride ? stride < o.stride : box < o.box;
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
    const Key key{p, rows, cols, stride, box_rows};
    auto it = cache.find(key);
    if (it == cache.end()) {
        if (cache.size() > 8192) cache.clear();
        CUtensorMap m;
        const cuuint64_t gdim[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
        const cuuint64_t gstride[1] = {(cuuint64_t)stride * 2};
        const cuuint32_t box[2] = {(cuuint32_t)TCG_K, (cuuint32_t)box_rows};
        const cuuint32_t estride[2] = {1, 1};
        if (encode(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(p), gdim, gstride, box, estride, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
            return cudaErrorInvalidValue;
        it = cache.emplace(key, m).first;
    }
    *out = it->second;
    return cudaSuccess;
}

// How a product is cut: the token tile (32 .. 256 columns) and the number of K runs whose estimated time is least.  Times are
// in steps of 64 columns at 256 tokens.  A step costs its products (an instruction narrower than 128 tokens takes as long as
// one of 128) or its bytes, whichever is more; an item adds fixed work and its epilogue, a cut tile writes and reads its sums.
struct TcgPlan {
    int nt, ksplit, stages;
};
TcgPlan tcg_plan(const tsb_ctx* ctx, int row_tiles, int units, int tokens) {
    TcgPlan best{256, 1, 4};
    float best_cost = 1e30f;
    const int sms = ctx->sm_count > 0 ? ctx->sm_count : 148;
    for (int nt : {32, 64, 128, 256}) {
        const int tok_tiles = (tokens + nt - 1) / nt;
        if (nt > 32 && nt / 2 >= tokens) continue;  // half of the tile would stand empty
        for (int ks = 1; ks <= TCG_MAX_SPLITS && ks <= units; ks++) {
            const int run = (units + ks - 1) / ks;
            if ((units + run - 1) / run != ks) continue;  // no empty runs
            if (ks > 1 && row_tiles * tok_tiles > TCG_TICKETS) continue;
            if (ks > 1 && (int64_t)row_tiles * tok_tiles * ks > 2 * sms) break;
            const float step = std::max(nt <= 128 ? 0.75f : 1.f, (128.f + nt) / 384.f * 1.1f);
            const float item = run * step + 6.f + (ks > 1 ? nt / 16.f * (1.f + 0.5f * ks) : nt / 64.f);
            const int waves = (row_tiles * tok_tiles * ks + sms - 1) / sms;
            const float cost = waves * item;
            if (cost < best_cost - 1e-3f) best_cost = cost, best.nt = nt, best.ksplit = ks;
        }
    }
    if (const char* env = getenv("TSB_PLAIN_PLAN")) {  // "tokens per tile,runs": experiments
        int nt = 0, ks = 0;
        if (sscanf(env, "%d,%d", &nt, &ks) == 2 && (nt == 32 || nt == 64 || nt == 128 || nt == 256) && ks >= 1 && ks <= TCG_MAX_SPLITS && ks <= units) {
            const int run = (units + ks - 1) / ks, tt = (tokens + nt - 1) / nt;
            ks = (units + run - 1) / run;
            if (ks == 1 || (int64_t)row_tiles * tt * ks <= 2 * sms) best.nt = nt, best.ksplit = ks;
        }
    }
    best.stages = std::min(TCG_MAX_STAGES, (TCG_SMEM_CAP - TCG_HEADER) / ((TCG_M + best.nt) * 128));
    return best;
}

template <int NT, int MT, int WK>
cudaError_t launch_few(tsb_ctx* ctx, cudaStream_t st, const PlainMat& w, const __nv_bfloat16* x, const __nv_bfloat16* x2, int64_t x_stride, int tokens,
                       const PlainEpi& epi) {
    // Not launched ahead of the attention kernel's end (the output product follows it): CTAs that become resident beside the
    // last attention CTAs are packed on few SMs and run with their small L1 - 67 to 75 us instead of 27 at 4096 x 18432.
    const bool ahead = epi.kind != PLAIN_ADD;
    const dim3 grid((unsigned)(w.rows / (16 * MT * (FEW_WARPS / WK))), (unsigned)((tokens + 8 * NT - 1) / (8 * NT)));
    return tsb_launch(ctx, plain_few_kernel<NT, MT, WK, false>, grid, dim3(FEW_WARPS * 32), 0, st, ahead,
                      (const __nv_bfloat16*)w.data, (int)w.cols, w.group_rows, w.group_cols, x, x2, x_stride, tokens, epi, PlainExperts{}, ctx->dev_error);
}
template <int NT, int WK>
cudaError_t launch_few_experts(tsb_ctx* ctx, cudaStream_t st, const PlainMat& w, const __nv_bfloat16* x, int64_t x_stride, const PlainExperts& ex, const PlainEpi& epi) {
    const dim3 grid((unsigned)(w.rows / (16 * (FEW_WARPS / WK))), (unsigned)expert_chunks_max(ex.slots, ex.n, ex.chunk_slots));
    return tsb_launch(ctx, plain_few_kernel<NT, 1, WK, true>, grid, dim3(FEW_WARPS * 32), 0, st, true, (const __nv_bfloat16*)w.data, (int)w.cols, 0, 0, x, x, x_stride,
                      0, epi, ex, ctx->dev_error);
}
template <int NT>
cudaError_t launch_few_experts_any(tsb_ctx* ctx, cudaStream_t st, const PlainMat& w, const __nv_bfloat16* x, int64_t x_stride, const PlainExperts& ex, const PlainEpi& epi) {
    const int units = (int)(w.cols / TCG_K);
    if (units == 1) return launch_few_experts<NT, 1>(ctx, st, w, x, x_stride, ex, epi);
    if (units < 4) return launch_few_experts<NT, 2>(ctx, st, w, x, x_stride, ex, epi);
    if (units < 8) return launch_few_experts<NT, 4>(ctx, st, w, x, x_stride, ex, epi);
    return launch_few_experts<NT, 8>(ctx, st, w, x, x_stride, ex, epi);
}

constexpr int FEW_MAX = 16;  // token rows up to which the weight-streaming kernel runs
// A product with few columns (one head's worth) is too short for the tensor-memory pipeline: the weight-streaming kernel takes it
// sixteen tokens at a time, its weights coming from the L2 cache after the first.
constexpr int FEW_SHORT_UNITS = 8, FEW_SHORT_MAX = 128;
constexpr int64_t FEW_SHORT_BYTES = 8 << 20;  // of weights, read once per sixteen tokens
template <int NT>
cudaError_t launch_few_any(tsb_ctx* ctx, cudaStream_t st, const PlainMat& w, const __nv_bfloat16* x, const __nv_bfloat16* x2, int64_t x_stride, int tokens,
                           const PlainEpi& epi) {
    const int units = (int)(w.cols / TCG_K);
    if (units == 1) return launch_few<NT, 1, 1>(ctx, st, w, x, x2, x_stride, tokens, epi);
    if (units < 4) return launch_few<NT, 1, 2>(ctx, st, w, x, x2, x_stride, tokens, epi);
    if (units < 8) return launch_few<NT, 1, 4>(ctx, st, w, x, x2, x_stride, tokens, epi);
    // two row tiles per CTA halve the activation reads when there are rows enough
    if (w.rows / 32 >= 4 * ctx->sm_count) return launch_few<NT, 2, 8>(ctx, st, w, x, x2, x_stride, tokens, epi);
    return launch_few<NT, 1, 8>(ctx, st, w, x, x2, x_stride, tokens, epi);
}

}  // namespace

size_t plain_gemm_workspace_bytes(const tsb_ctx* ctx) {
    const int sms = ctx->sm_count > 0 ? ctx->sm_count : 148;
    return TCG_TICKETS * sizeof(uint32_t) + (size_t)(2 * sms) * TCG_M * TCG_NMAX * sizeof(float);
}

cudaError_t launch_plain_gemm(tsb_ctx* ctx, cudaStream_t st, bool f32, const PlainMat& w, const void* x, const void* x2, int64_t x_stride, int x_rows,
                              int tokens, const PlainEpi& epi, void* workspace) {
    if (tokens <= 0) return cudaSuccess;
    if (f32) {
        dim3 grid((unsigned)(w.rows / F32_TILE), (unsigned)((tokens + F32_TILE - 1) / F32_TILE));
        return tsb_launch(ctx, plain_f32_kernel<false>, grid, dim3(256), 0, st, true, (const float*)w.data, (int)w.cols, w.group_rows, w.group_cols,
                          (const float*)x, (const float*)x2, x_stride, tokens, epi, PlainExperts{}, ctx->dev_error);
    }
    const __nv_bfloat16 *xb = (const __nv_bfloat16*)x, *xb2 = (const __nv_bfloat16*)x2;
    if (tokens <= FEW_MAX || (tokens <= FEW_SHORT_MAX && w.cols <= FEW_SHORT_UNITS * TCG_K && w.rows * w.cols * 2 * ((tokens + 15) / 16) <= FEW_SHORT_BYTES))
        return tokens <= 8 ? launch_few_any<1>(ctx, st, w, xb, xb2, x_stride, tokens, epi) : launch_few_any<2>(ctx, st, w, xb, xb2, x_stride, tokens, epi);
    const int row_tiles = (int)(w.rows / TCG_M), units = (int)(w.cols / TCG_K);
    const TcgPlan p = tcg_plan(ctx, row_tiles, units, tokens);
    CUtensorMap wm, xm, xm2;
    cudaError_t e = tcg_map(w.data, w.rows, w.cols, w.cols, TCG_M, &wm);
    const int64_t x_cols = w.group_rows ? (w.rows / w.group_rows - 1) * w.group_cols + w.cols : w.cols;
    if (e == cudaSuccess) e = tcg_map(x, x_rows, x_cols, x_stride, p.nt, &xm);
    if (e == cudaSuccess) e = tcg_map(x2 ? x2 : x, x_rows, x_cols, x_stride, p.nt, &xm2);
    if (e != cudaSuccess) return e;
    const int tok_tiles = (tokens + p.nt - 1) / p.nt;
    const int items = row_tiles * tok_tiles * p.ksplit;
    uint32_t* tickets = static_cast<uint32_t*>(workspace);
    float* part = reinterpret_cast<float*>(tickets + TCG_TICKETS);
    const size_t smem = TCG_HEADER + (size_t)p.stages * (TCG_M + p.nt) * 128;
    auto run = [&](auto kernel, SmemOptIn& configured) {
        if (cudaError_t r = tsb_opt_in_smem(ctx, kernel, (size_t)TCG_SMEM_CAP, configured); r != cudaSuccess) return r;
        return tsb_launch(ctx, kernel, dim3((unsigned)std::min(items, ctx->sm_count)), dim3(TCG_THREADS), smem, st, true, wm, xm, xm2, row_tiles, tok_tiles,
                          units, p.ksplit, p.nt, p.stages, tokens, w.group_rows, w.group_cols, epi, PlainExperts{}, part, tickets, ctx->dev_error);
    };
    static SmemOptIn configured[3];
    if (epi.kind == PLAIN_STORE) return run(plain_tc_kernel<PLAIN_STORE, false>, configured[0]);
    if (epi.kind == PLAIN_ADD) return run(plain_tc_kernel<PLAIN_ADD, false>, configured[1]);
    return run(plain_tc_kernel<PLAIN_MIXER, false>, configured[2]);
}

cudaError_t launch_plain_gemm_experts(tsb_ctx* ctx, cudaStream_t st, bool f32, bool tensor, const PlainMat& w, const void* x, int64_t x_stride, int x_rows,
                                      const PlainExperts& ex, const PlainEpi& epi) {
    if (ex.slots <= 0) return cudaSuccess;
    if (ex.n > EXPERTS_MAX || epi.kind != PLAIN_MIXER) return cudaErrorInvalidValue;
    if (f32) {
        const dim3 grid((unsigned)(w.rows / F32_TILE), (unsigned)expert_chunks_max(ex.slots, ex.n, ex.chunk_slots));
        return tsb_launch(ctx, plain_f32_kernel<true>, grid, dim3(256), 0, st, true, (const float*)w.data, (int)w.cols, 0, 0, (const float*)x, (const float*)x, x_stride, 0,
                          epi, ex, ctx->dev_error);
    }
    const __nv_bfloat16* xb = (const __nv_bfloat16*)x;
    if (!tensor)
        return ex.chunk_slots <= 8 ? launch_few_experts_any<1>(ctx, st, w, xb, x_stride, ex, epi) : launch_few_experts_any<2>(ctx, st, w, xb, x_stride, ex, epi);
    if (ex.token_of) return cudaErrorInvalidValue;
    const int row_tiles = (int)(w.rows / TCG_M), units = (int)(w.cols / TCG_K);
    int nt = 32;  // a tile that holds an expert's slots when they are spread evenly, with some room
    while (nt < TCG_NMAX && nt < ex.slots / ex.n * 5 / 4) nt *= 2;
    const int stages = std::min(TCG_MAX_STAGES, (TCG_SMEM_CAP - TCG_HEADER - TCG_EXPERT_BYTES) / ((TCG_M + nt) * 128));
    CUtensorMap wm, xm;
    cudaError_t e = tcg_map(w.data, w.rows * ex.n, w.cols, w.cols, TCG_M, &wm);
    if (e == cudaSuccess) e = tcg_map(x, x_rows, w.cols, x_stride, nt, &xm);
    if (e != cudaSuccess) return e;
    const size_t smem = TCG_HEADER + (size_t)stages * (TCG_M + nt) * 128 + TCG_EXPERT_BYTES;
    static SmemOptIn configured;
    if ((e = tsb_opt_in_smem(ctx, plain_tc_kernel<PLAIN_MIXER, true>, (size_t)TCG_SMEM_CAP, configured)) != cudaSuccess) return e;
    const int64_t items = (int64_t)(ex.slots / nt + std::min(ex.n, ex.slots)) * row_tiles;
    return tsb_launch(ctx, plain_tc_kernel<PLAIN_MIXER, true>, dim3((unsigned)std::min<int64_t>(items, ctx->sm_count)), dim3(TCG_THREADS), smem, st, true, wm, xm, xm,
                      row_tiles, 1, units, 1, nt, stages, 0, 0, 0, epi, ex, (float*)nullptr, (uint32_t*)nullptr, ctx->dev_error);
}
