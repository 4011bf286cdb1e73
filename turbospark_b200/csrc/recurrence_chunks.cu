// Recurrent mixers over long portions, REC_CHUNK rows at a time, bfloat16 operands on mma.sync with f32 accumulators.
//
// With E_t the product of a chunk's decays up to row t and S the state before the chunk,
//   o_t = E_t q_t . S + sum_{s <= t} (E_t / E_s) (q_t . k_s) v_s,    S' = E_T S + sum_s (E_T / E_s) k_s v_s^T.
// Three launches: what every chunk adds to the state (all chunks at once), the states before the chunks (a walk over the chunks, element by
// element), the outputs (all chunks at once).  A CTA of the first and the last has one chunk, one head and 64 or 128 value columns.
//
// What is f32 stays f32-like: an operand that is not a projection (state, weighted products, decayed queries, keys or values) goes into a
// product as the sum of two bfloat16 numbers, which keeps 16 bits of it.
//
// Decay per head (REC_MLSTM, REC_SSD): E is a number per row; the ratios are exponentials of differences of its logarithm, applied to the
// products of plain queries and keys, and to the values on their way into the state.
// Decay per row of the state (REC_FORGET): E is a vector.  Into the state go keys times E_T / E_s, a product over the rows behind s; queries take
// E_t, keys 1 / E_s, both shifted by 2^60 to use the whole range of exponents.  1 / E grows, so where a component of E falls below 2^-140
// the chunk is cut: rows behind a cut meet each other with E counted from the cut, and the rows before it with keys brought to the cut.
#include <algorithm>

#include "mma_dev.cuh"
#include "recurrence_dev.cuh"

namespace {

constexpr int C = REC_CHUNK, THREADS = 256;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float E_ONE = 1152921504606846976.f, E_MIN = 8.2718061e-25f;  // 2^60 stands for E = 1, 2^-80 for the least E

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.f + __expf(-z)); }
__device__ __forceinline__ uint32_t pack(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
// two numbers as the sum of two bfloat16 pairs
__device__ __forceinline__ void split(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack(a, b);
    lo = pack(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xFFFF0000u));
}
// byte offset of 16-byte piece p of row r; rows of BYTES (a multiple of 128), pieces permuted so that eight rows' worth of one piece spread
// over all banks
template <int BYTES>
__device__ __forceinline__ uint32_t at(int r, int p) {
    return (uint32_t)(r * BYTES + ((p ^ (r & 7)) << 4));
}

// ---- what the launches leave for each other, per (chunk, head)
struct Scratch {
    float* add;     // [dim][vdim]: what the chunk adds; after the walk the state before it, four numbers as four high and four low halves
    float* norm;    // REC_MLSTM: the same for the normaliser, [dim]
    float* decay;   // REC_FORGET: E_T [dim]; REC_SSD: E_T; REC_MLSTM: log E_T, and the maximum the chunk's part is relative to
    double* top;    // REC_MLSTM: the running maximum before the chunk
    float4* rows;   // decay per head: input scales and log E of rows 2 l and 2 l + 1, [32]
};
__host__ __device__ inline int decay_width(int kind, int dim) { return kind == REC_FORGET ? dim : 2; }
size_t align16(size_t n) { return (n + 15) / 16 * 16; }
Scratch scratch_of(const Recurrence& r, void* p, int chunks) {
    const size_t n = (size_t)chunks * r.heads;
    Scratch s;
    uint8_t* b = static_cast<uint8_t*>(p);
    s.add = reinterpret_cast<float*>(b), b += align16(n * r.dim * r.vdim * 4);
    s.norm = reinterpret_cast<float*>(b), b += align16(r.kind == REC_MLSTM ? n * r.dim * 4 : 0);
    s.decay = reinterpret_cast<float*>(b), b += align16(n * decay_width(r.kind, r.dim) * 4);
    s.top = reinterpret_cast<double*>(b), b += align16(n * 8);
    s.rows = reinterpret_cast<float4*>(b);
    return s;
}

// rows x columns of a projection into shared memory, zeros outside
template <int ROW_BYTES, int NT>
__device__ __forceinline__ void copy_tile(uint32_t dst, const __nv_bfloat16* src, int64_t stride, int n_rows, int n_cols) {
    for (int i = threadIdx.x; i < C * (ROW_BYTES / 16); i += NT) {
        const int r = i / (ROW_BYTES / 16), c = i % (ROW_BYTES / 16);
        const bool ok = r < n_rows && c * 8 < n_cols;
        cp16(dst + at<ROW_BYTES>(r, c), src + (ok ? r * stride + c * 8 : 0), ok);
    }
}

// Gates of a chunk, by warp 0: lane l has rows 2 l and 2 l + 1.
struct RowGates {
    float in[2], log_e[2], end;  // SSD: step; MLSTM: log input gate.  log E up to the row, and at the chunk's end
};
template <int KIND>
__device__ __forceinline__ RowGates row_gates(const Recurrence& a, int row0, int n, int head, int lane) {
    RowGates g;
    const float rate = KIND == REC_SSD ? expf(a.a_log[head]) : 0.f;
    float d[2];
#pragma unroll
    for (int i = 0; i < 2; i++) {
        const int r = 2 * lane + i;
        float2 v = make_float2(KIND == REC_MLSTM ? -1e30f : 0.f, 0.f);
        if (r < n) v = KIND == REC_MLSTM ? mlstm_gates(a, row0 + r, head) : ssd_gates(a, row0 + r, head, rate);
        g.in[i] = v.x, d[i] = v.y;
    }
    float sum = d[0] + d[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += v;
    }
    g.log_e[1] = sum, g.log_e[0] = sum - d[1], g.end = __shfl_sync(0xffffffffu, sum, 31);
    return g;
}

// REC_FORGET: a thread has two neighbouring channels, 2 (thread % (DK / 2)), of TR rows.
template <int DK, int NT>
struct Channels {
    static constexpr int RS = NT / (DK / 2), TR = C / RS;  // row splits, rows of a thread
    int ch, part, first;
    __device__ __forceinline__ Channels() : ch(threadIdx.x % (DK / 2) * 2), part(threadIdx.x / (DK / 2)), first(part * TR) {}
    // of the split i and the thread's channels
    __device__ __forceinline__ float2& total(float* fv, int i) const { return reinterpret_cast<float2*>(fv)[i * (DK / 2) + ch / 2]; }
    __device__ __forceinline__ uint32_t key(int r) const { return at<DK * 2>(r, ch >> 3) + (ch & 7) * 2; }
};
// 1 - f = (1 - l) sigmoid(-z)
__device__ __forceinline__ float one_minus_f(float z, float open) {
    const float e = __expf(-fabsf(z)), d = __fdividef(1.f, 1.f + e);
    return open * (z >= 0.f ? e * d : d);
}
template <int DK>
__device__ __forceinline__ float2 open_of(const Recurrence& a, int head, int ch) {  // 1 - l; channels outside stay open
    const float* l = a.lower + (int64_t)head * a.dim + ch;
    return ch < a.dim ? make_float2(1.f - l[0], 1.f - l[1]) : make_float2(0.f, 0.f);
}
// pre: pre-activations of the chunk in shared memory, which become 1 - f; returns the products of the thread's f.
template <int DK, int NT>
__device__ __forceinline__ float2 forget_gates(const Recurrence& a, float* pre, int head, int n) {
    const Channels<DK, NT> me;
    const float2 open = open_of<DK>(a, head, me.ch);
    float2 product = make_float2(1.f, 1.f);
#pragma unroll 4
    for (int i = 0; i < me.TR; i++) {
        float2& x = *reinterpret_cast<float2*>(pre + (me.first + i) * DK + me.ch);
        const bool in = me.first + i < n;
        x = in ? make_float2(one_minus_f(x.x, open.x), one_minus_f(x.y, open.y)) : make_float2(0.f, 0.f);
        product.x *= 1.f - x.x, product.y *= 1.f - x.y;
    }
    return product;
}
template <int DK, int NT>
__device__ __forceinline__ void copy_gates(const Recurrence& a, uint32_t dst, int row0, int n, int head) {
    const float* gz = a.gate + (int64_t)row0 * a.gate_stride + (int64_t)head * a.dim;
    for (int i = threadIdx.x; i < C * (DK / 4); i += NT) {
        const int r = i / (DK / 4), c = i % (DK / 4);
        const bool ok = r < n && c * 4 < a.dim;
        cp16(dst + (r * DK + c * 4) * 4, gz + (ok ? r * a.gate_stride + c * 4 : 0), ok);
    }
}
__device__ __forceinline__ void put_split(uint8_t* hi, uint8_t* lo, uint32_t off, float a, float b) {
    uint32_t h, l;
    split(a, b, h, l);
    *reinterpret_cast<uint32_t*>(hi + off) = h;
    *reinterpret_cast<uint32_t*>(lo + off) = l;
}

// ------------------------------------------------------------------ what a chunk adds to the state
template <int KIND, int DK, int VB>
struct AddSmem {
    static constexpr bool FORGET = KIND == REC_FORGET;
    static constexpr int KEY = C * DK * 2, VAL = C * VB * 2;  // a tile of keys, of values
    static constexpr int K = 0, V = FORGET ? 2 * KEY : KEY, W = V + VAL;  // FORGET: keys, values; else keys, values, weighted values (high, low)
    static constexpr int Z = W, F = FORGET ? Z + C * DK * 4 : W + 2 * VAL;
    static constexpr int BYTES = F + (FORGET ? 2 * THREADS : C + 4) * 4;
};

template <int KIND, int DK, int VB>
__global__ void __launch_bounds__(THREADS)
    chunk_add_kernel(const __grid_constant__ Recurrence a, const __grid_constant__ RowTiles chunks, const __grid_constant__ Scratch out, uint32_t* __restrict__ err) {
    using M = AddSmem<KIND, DK, VB>;
    constexpr int BV = VB * 2;
    constexpr bool FORGET = KIND == REC_FORGET, MLSTM = KIND == REC_MLSTM;
    constexpr int KB = DK * 2, MT = DK / 16, SPLIT = MT < 8 ? 8 / MT : 1, MS = MT < 8 ? 1 : MT / 8, NV = VB / 8 / SPLIT;
    extern __shared__ __align__(128) uint8_t smem[];
    const uint32_t base = smem_u32(smem);
    float* fv = reinterpret_cast<float*>(smem + M::F);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int head = blockIdx.y, col0 = blockIdx.x * VB;
    const AttnTile tile = row_tile(chunks, blockIdx.z);
    const int row0 = tile.row_first, n = min(tile.n_rows, C);
    const int64_t slot = (int64_t)blockIdx.z * a.heads + head;
    const __nv_bfloat16* gv = static_cast<const __nv_bfloat16*>(a.v) + (int64_t)row0 * a.v_stride + (int64_t)head * a.vdim + col0;
    pdl_wait();
    pdl_launch_dependents();
    copy_tile<BV, THREADS>(base + M::V, gv, a.v_stride, n, a.vdim - col0);
    if (FORGET) {
        copy_gates<DK, THREADS>(a, base + M::Z, row0, n, head);
    } else {
        copy_tile<KB, THREADS>(base + M::K, static_cast<const __nv_bfloat16*>(a.k) + (int64_t)row0 * a.k_stride + head / a.heads_per_key * a.dim, a.k_stride, n, a.dim);
    }
    cp_async_commit();
    if (!FORGET && warp == 0) {
        // weights of the rows: E_T / E_s times the input scale (MLSTM: relative to the largest of them)
        const RowGates g = row_gates<FORGET ? REC_SSD : KIND>(a, row0, n, head, lane);
        float w[2], rel = 0.f;
        if (MLSTM) {
            w[0] = g.end - g.log_e[0] + g.in[0], w[1] = g.end - g.log_e[1] + g.in[1];
            rel = fmaxf(w[0], w[1]);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) rel = fmaxf(rel, __shfl_xor_sync(0xffffffffu, rel, o));
            w[0] = ex2((w[0] - rel) * LOG2E), w[1] = ex2((w[1] - rel) * LOG2E);
        } else {
            w[0] = ex2((g.end - g.log_e[0]) * LOG2E) * g.in[0], w[1] = ex2((g.end - g.log_e[1]) * LOG2E) * g.in[1];
        }
        fv[2 * lane] = w[0], fv[2 * lane + 1] = w[1];
        if (blockIdx.x == 0) out.rows[slot * 32 + lane] = make_float4(g.in[0], g.in[1], g.log_e[0], g.log_e[1]);
        if (blockIdx.x == 0 && lane == 0) {
            out.decay[slot * 2] = MLSTM ? g.end : expf(g.end);
            out.decay[slot * 2 + 1] = rel;
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    if (FORGET) {
        float* pre = reinterpret_cast<float*>(smem + M::Z);
        const Channels<DK, THREADS> me;
        me.total(fv, me.part) = forget_gates<DK, THREADS>(a, pre, head, n);
        __syncthreads();
        float2 e = make_float2(1.f, 1.f);  // products of the rows behind
        for (int i = me.part + 1; i < me.RS; i++) e.x *= me.total(fv, i).x, e.y *= me.total(fv, i).y;
#pragma unroll 4
        for (int i = me.TR - 1; i >= 0; i--) {
            const int r = me.first + i;
            const float2 k = *reinterpret_cast<const float2*>(pre + r * DK + me.ch);
            put_split(smem + M::K, smem + M::K + M::KEY, me.key(r), k.x * e.x, k.y * e.y);
            e.x *= 1.f - k.x, e.y *= 1.f - k.y;
        }
        if (me.part == 0 && blockIdx.x == 0 && me.ch < a.dim) *reinterpret_cast<float2*>(out.decay + slot * a.dim + me.ch) = e;
    } else {
        for (int i = threadIdx.x; i < C * (VB / 2); i += THREADS) {
            const int r = i / (VB / 2), c = i % (VB / 2);
            const uint32_t off = at<BV>(r, c >> 2) + (c & 3) * 4, v = *reinterpret_cast<const uint32_t*>(smem + M::V + off);
            uint32_t hi, lo;
            split(__uint_as_float(v << 16) * fv[r], __uint_as_float(v & 0xFFFF0000u) * fv[r], hi, lo);
            *reinterpret_cast<uint32_t*>(smem + M::W + off) = hi;
            *reinterpret_cast<uint32_t*>(smem + M::W + M::VAL + off) = lo;
        }
        if (MLSTM && blockIdx.x == 0)
            for (int c = threadIdx.x; c < a.dim; c += THREADS) {
                float x = 0.f;
#pragma unroll 8
                for (int r = 0; r < C; r++)
                    x = fmaf(fv[r], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(smem + M::K + at<KB>(r, c >> 3) + (c & 7) * 2)), x);
                out.norm[slot * a.dim + c] = x;
            }
    }
    __syncthreads();
    // keys (transposed) times values: m-tile per warp, or half of the columns of one
    const int m0 = MT < 8 ? warp % MT : warp, nv0 = MT < 8 ? warp / MT * NV : 0;
    float s[MS][NV][4] = {};
    const uint32_t vh = base + (FORGET ? M::V : M::W);
#pragma unroll
    for (int ks = 0; ks < C / 16; ks++) {
        uint32_t bh[NV / 2][4], bl[NV / 2][4];
#pragma unroll
        for (int np = 0; np < NV / 2; np++) {
            ldsm4_t(bh[np], vh + at<BV>(ks * 16 + (lane & 15), nv0 + np * 2 + (lane >> 4)));
            if (!FORGET) ldsm4_t(bl[np], vh + M::VAL + at<BV>(ks * 16 + (lane & 15), nv0 + np * 2 + (lane >> 4)));
        }
#pragma unroll
        for (int m = 0; m < MS; m++) {
            const int c8 = (m0 + 8 * m) * 2 + ((lane >> 3) & 1), r = ks * 16 + (lane & 7) + ((lane >> 4) << 3);
            uint32_t kh[4], kl[4];
            ldsm4_t(kh, base + M::K + at<KB>(r, c8));
            if (FORGET) ldsm4_t(kl, base + M::K + M::KEY + at<KB>(r, c8));
#pragma unroll
            for (int np = 0; np < NV / 2; np++) {
                mma_bf16(s[m][2 * np], kh, bh[np][0], bh[np][1]), mma_bf16(s[m][2 * np + 1], kh, bh[np][2], bh[np][3]);
                if (FORGET) mma_bf16(s[m][2 * np], kl, bh[np][0], bh[np][1]), mma_bf16(s[m][2 * np + 1], kl, bh[np][2], bh[np][3]);
                else mma_bf16(s[m][2 * np], kh, bl[np][0], bl[np][1]), mma_bf16(s[m][2 * np + 1], kh, bl[np][2], bl[np][3]);
            }
        }
    }
    float* dst = out.add + slot * a.dim * a.vdim;
#pragma unroll
    for (int m = 0; m < MS; m++)
#pragma unroll
        for (int i = 0; i < NV; i++)
#pragma unroll
            for (int h = 0; h < 2; h++) {
                const int r = (m0 + 8 * m) * 16 + gid + 8 * h, c = col0 + (nv0 + i) * 8 + 2 * tig;
                if (r < a.dim && c < a.vdim) *reinterpret_cast<float2*>(dst + (int64_t)r * a.vdim + c) = make_float2(s[m][i][2 * h], s[m][i][2 * h + 1]);
            }
}

// ------------------------------------------------------------------ states before the chunks
// A thread owns four neighbouring numbers of a head's state and walks the chunks of the portion.  The running maximum after the portion is left to
// the next launch: every thread reads the one before it.
template <int KIND>
__global__ void __launch_bounds__(THREADS, 4)
    chunk_walk_kernel(const __grid_constant__ Recurrence a, const __grid_constant__ RecurrenceChunks c, const __grid_constant__ Scratch s, uint32_t* __restrict__ err) {
    constexpr bool FORGET = KIND == REC_FORGET, MLSTM = KIND == REC_MLSTM;
    const int per_seq = (c.rows_per_seq + C - 1) / C;
    const ChunkPortion p = c.portions ? c.portions[blockIdx.z] : ChunkPortion{(int)blockIdx.z * c.rows_per_seq, c.rows_per_seq, (int)blockIdx.z * per_seq};
    const tsb_row_desc rd = a.rows[p.first_row];
    const int head = blockIdx.y, pos0 = rd.base + rd.slot, n = (p.n_rows + C - 1) / C;
    const int state4 = a.dim * a.vdim / 4, i4 = blockIdx.x * THREADS + threadIdx.x;
    const int norm_i = i4 - state4;  // MLSTM: threads behind the state take a number of the normaliser each
    if (rd.seq < 0 || rd.seq >= a.state.n_streams) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        pdl_wait();
        return;
    }
    const bool is_norm = MLSTM && norm_i >= 0 && norm_i < a.dim;
    const int64_t from = rec_slot(a, rd.seq, pos0 - 1) * a.heads + head, to = rec_slot(a, rd.seq, pos0 + p.n_rows - 1) * a.heads + head;
    const int64_t head_state = (int64_t)a.dim * a.vdim;
    const int copies = recurrence_copies(a.vdim);
    const int row = i4 < state4 ? i4 * 4 / a.vdim : 0;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    double top = 0.0;
    if (pos0 > 0) {
        if (i4 < state4) v = *reinterpret_cast<const float4*>(a.state.s + from * head_state + (int64_t)i4 * 4);
        if (is_norm) v.x = a.state.norm[from * copies * a.dim + norm_i];
        if (MLSTM) top = a.state.top[from * copies];
    }
    pdl_wait();
    pdl_launch_dependents();
    if (i4 >= state4 && !is_norm) return;
    constexpr int AHEAD = 4;
    const int width = FORGET ? a.dim : 2;
    float4 next[AHEAD];
    float2 gate[AHEAD];
    auto fetch = [&](int k, float4& x, float2& g) {
        const int64_t slot = (int64_t)(p.first_chunk + k) * a.heads + head;
        if (is_norm) x.x = s.norm[slot * a.dim + norm_i];
        else x = *reinterpret_cast<const float4*>(s.add + slot * head_state + (int64_t)i4 * 4);
        if (FORGET) g.x = s.decay[slot * width + row];
        else g = *reinterpret_cast<const float2*>(s.decay + slot * width);
    };
#pragma unroll
    for (int k = 0; k < AHEAD; k++)
        if (k < n) fetch(k, next[k], gate[k]);
    for (int k0 = 0; k0 < n; k0 += AHEAD) {
#pragma unroll
        for (int j = 0; j < AHEAD; j++) {
            const int k = k0 + j;
            if (k >= n) break;
            const float4 add = next[j];
            const float2 g = gate[j];
            if (k + AHEAD < n) fetch(k + AHEAD, next[j], gate[j]);
            const int64_t slot = (int64_t)(p.first_chunk + k) * a.heads + head;
            if (is_norm) {
                s.norm[slot * a.dim + norm_i] = v.x;
                if (norm_i == 0) s.top[slot] = top;
            } else {
                uint4 w;
                split(v.x, v.y, w.x, w.z);
                split(v.z, v.w, w.y, w.w);
                *reinterpret_cast<uint4*>(s.add + slot * head_state + (int64_t)i4 * 4) = w;
            }
            float keep = g.x, write = 1.f;
            if (MLSTM) {
                const double old = top + g.x, m = fmax(old, (double)g.y);
                keep = expf((float)(old - m)), write = expf((float)(g.y - m));
                top = m;
            }
            v.x = fmaf(keep, v.x, write * add.x), v.y = fmaf(keep, v.y, write * add.y), v.z = fmaf(keep, v.z, write * add.z), v.w = fmaf(keep, v.w, write * add.w);
        }
    }
    if (is_norm) {
        for (int k = 0; k < copies; k++) a.state.norm[(to * copies + k) * a.dim + norm_i] = v.x;
    } else {
        *reinterpret_cast<float4*>(a.state.s + to * head_state + (int64_t)i4 * 4) = v;
    }
}

// ------------------------------------------------------------------ outputs of a chunk
template <int KIND, int DK, int VB, int NT>
struct OutSmem {
    static constexpr bool FORGET = KIND == REC_FORGET;
    static constexpr int KEY = C * DK * 2, VAL = C * VB * 2, STATE = DK * VB * 2, PROD = C * C * 2;
    // queries and keys (FORGET: high and low parts of each), values, state (high, low); products (high, low) where the keys were, or from there on
    static constexpr int Q = 0, K = FORGET ? 2 * KEY : KEY, KEYS = (FORGET ? 2 : 1) * KEY > 2 * PROD ? (FORGET ? 2 : 1) * KEY : 2 * PROD;
    static constexpr int V = K + KEYS, S = V + VAL, P = K, F = S + 2 * STATE;
    static constexpr int Z = S;  // FORGET: the gates of the chunk, before the state takes their place
    static_assert(!FORGET || C * DK * 4 <= 2 * STATE, "");
    static constexpr int BYTES = F + (FORGET ? 2 * NT : KIND == REC_MLSTM ? 4 * C + DK + 5 * C : 3 * C) * 4;
};

// NT threads: a warp per 16 rows and 32 value columns
template <int KIND, int DK, int VB, int NT>
__global__ void __launch_bounds__(NT, NT > 256 ? 1 : DK > 128 || KIND == REC_FORGET ? 2 : 3)
    chunk_out_kernel(const __grid_constant__ Recurrence a, const __grid_constant__ RowTiles chunks, const __grid_constant__ Scratch in, uint32_t* __restrict__ err) {
    using M = OutSmem<KIND, DK, VB, NT>;
    static_assert(NT / 32 == 4 * (VB / 32), "");
    constexpr bool FORGET = KIND == REC_FORGET, MLSTM = KIND == REC_MLSTM, SSD = KIND == REC_SSD;
    constexpr int KB = DK * 2, BV = VB * 2, KS = DK / 16, NV = 4, NW = NT / 32;
    extern __shared__ __align__(128) uint8_t smem[];
    const uint32_t base = smem_u32(smem);
    float* fv = reinterpret_cast<float*>(smem + M::F);
    float *ea = fv, *eb = fv + C, *gain = fv + 2 * C, *floor_ = fv + 3 * C, *norm = fv + 4 * C, *nq = norm + DK;  // nq [rows][5]: shares of n . q
    __shared__ int cut_end;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int head = blockIdx.y, col0 = blockIdx.x * VB, key_at = head / a.heads_per_key * a.dim;
    const AttnTile tile = row_tile(chunks, blockIdx.z);
    const int row0 = tile.row_first, n = min(tile.n_rows, C);
    const int64_t slot = (int64_t)blockIdx.z * a.heads + head;
    const __nv_bfloat16* gq = static_cast<const __nv_bfloat16*>(a.q) + (int64_t)row0 * a.q_stride + key_at;
    pdl_wait();
    pdl_launch_dependents();
    copy_tile<BV, NT>(base + M::V, static_cast<const __nv_bfloat16*>(a.v) + (int64_t)row0 * a.v_stride + (int64_t)head * a.vdim + col0, a.v_stride, n, a.vdim - col0);
    copy_tile<KB, NT>(base + M::Q, gq, a.q_stride, n, a.dim);
    if (FORGET) {
        copy_gates<DK, NT>(a, base + M::Z, row0, n, head);
    } else {
        copy_tile<KB, NT>(base + M::K, static_cast<const __nv_bfloat16*>(a.k) + (int64_t)row0 * a.k_stride + key_at, a.k_stride, n, a.dim);
    }
    // the state: four numbers as four high and four low halves, to two tiles
    constexpr int PIECES = DK * (VB / 4), MINE = PIECES / NT;
    const float* src = in.add + slot * a.dim * a.vdim + col0;
    uint4 held[FORGET ? MINE : 1];  // FORGET: their place is still taken
#pragma unroll
    for (int k = 0; k < MINE; k++) {
        const int i = k * NT + threadIdx.x, r = i / (VB / 4), c = i % (VB / 4);
        const bool ok = r < a.dim && col0 + c * 4 < a.vdim;
        const float* p = ok ? src + (int64_t)r * a.vdim + c * 4 : in.add;
        if (FORGET) {
            held[FORGET ? k : 0] = ok ? *reinterpret_cast<const uint4*>(p) : make_uint4(0, 0, 0, 0);
        } else {
            const uint32_t off = base + M::S + at<BV>(r, c >> 1) + (c & 1) * 8;
            cp8(off, p, ok), cp8(off + M::STATE, p + 2, ok);
        }
    }
    cp_async_commit();
    if (!FORGET) {
        if (MLSTM)
            for (int i = threadIdx.x; i < DK; i += NT) norm[i] = i < a.dim ? in.norm[slot * a.dim + i] : 0.f;
        if (warp == 0) {
            const float4 kept = in.rows[slot * 32 + lane];
            const RowGates g{{kept.x, kept.y}, {kept.z, kept.w}, __shfl_sync(0xffffffffu, kept.w, 31)};
            if (SSD) {
#pragma unroll
                for (int i = 0; i < 2; i++) ea[2 * lane + i] = g.log_e[i] * LOG2E, eb[2 * lane + i] = -g.log_e[i] * LOG2E, gain[2 * lane + i] = g.in[i];
            } else {
                // relative to the maximum before the chunk: i_s - F_s - m, and its running maximum with 0
                const double top = in.top[slot];
                const float b0 = (float)((double)g.in[0] - g.log_e[0] - top), b1 = (float)((double)g.in[1] - g.log_e[1] - top);
                float mx = fmaxf(b0, b1);
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const float v = __shfl_up_sync(0xffffffffu, mx, o);
                    if (lane >= o) mx = fmaxf(mx, v);
                }
                const float before = __shfl_up_sync(0xffffffffu, mx, 1);
                const float m1 = fmaxf(mx, 0.f), m0 = fmaxf(lane > 0 ? fmaxf(before, b0) : b0, 0.f);
                ea[2 * lane] = -m0 * LOG2E, ea[2 * lane + 1] = -m1 * LOG2E, eb[2 * lane] = b0 * LOG2E, eb[2 * lane + 1] = b1 * LOG2E;
                gain[2 * lane] = gain[2 * lane + 1] = 1.f;
                floor_[2 * lane] = expf(-(float)(top + g.log_e[0] + m0)), floor_[2 * lane + 1] = expf(-(float)(top + g.log_e[1] + m1));
                const tsb_row_desc rd = a.rows[row0 + n - 1];
                if (lane == 31 && blockIdx.x == 0 && (row0 + n >= a.n_rows || a.rows[row0 + n].seq != rd.seq)) {  // the portion's last row
                    const int copies = recurrence_copies(a.vdim);
                    double* to = a.state.top + (rec_slot(a, rd.seq, rd.base + rd.slot) * a.heads + head) * copies;
                    for (int k = 0; k < copies; k++) to[k] = top + g.end + m1;
                }
            }
        }
    }
    cp_async_wait<0>();
    __syncthreads();

    // ---- FORGET: queries times E_t, keys over E_s
    const Channels<FORGET ? DK : 64, NT> me;
    bool cuts = false;
    if (FORGET) {
        float* pre = reinterpret_cast<float*>(smem + M::Z);
        const float2 mine = forget_gates<DK, NT>(a, pre, head, n);
        me.total(fv, me.part) = mine;
        __syncthreads();
        float2 e = make_float2(E_ONE, E_ONE);  // E at the start of the thread's rows
        for (int i = 0; i < me.part; i++) e.x *= me.total(fv, i).x, e.y *= me.total(fv, i).y;
        cuts = __syncthreads_or(fminf(e.x * mine.x, e.y * mine.y) < E_MIN);  // E only falls
#pragma unroll 4
        for (int i = 0; i < me.TR; i++) {
            const int r = me.first + i;
            const float2 k = *reinterpret_cast<const float2*>(pre + r * DK + me.ch);
            e.x *= 1.f - k.x, e.y *= 1.f - k.y;
            const uint32_t off = me.key(r), x = *reinterpret_cast<const uint32_t*>(smem + M::Q + off);
            put_split(smem + M::Q, smem + M::Q + M::KEY, off, silu(__uint_as_float(x << 16)) * e.x, silu(__uint_as_float(x & 0xFFFF0000u)) * e.y);
            put_split(smem + M::K, smem + M::K + M::KEY, off, cuts ? 0.f : __fdividef(k.x, e.x), cuts ? 0.f : __fdividef(k.y, e.y));
        }
        __syncthreads();  // the gates have been read
#pragma unroll
        for (int k = 0; k < MINE; k++) {
            const int i = k * NT + threadIdx.x, r = i / (VB / 4), c = i % (VB / 4);
            const uint32_t off = at<BV>(r, c >> 1) + (c & 1) * 8;
            const uint4 w = held[FORGET ? k : 0];
            *reinterpret_cast<uint2*>(smem + M::S + off) = make_uint2(w.x, w.y);
            *reinterpret_cast<uint2*>(smem + M::S + M::STATE + off) = make_uint2(w.z, w.w);
        }
        __syncthreads();
    }

    const int mt = warp & 3, c8 = (warp >> 2) * NV;  // row tile, first column group
    const int ta = mt * 16 + gid, tb = ta + 8;
    float o[NV][4] = {};
    // ---- queries against the state
    {
        float share[2] = {0.f, 0.f};
#pragma unroll 4
        for (int ks = 0; ks < KS; ks++) {
            uint32_t qa[4], ql[4];
            ldsm4(qa, base + M::Q + at<KB>(mt * 16 + (lane & 15), ks * 2 + (lane >> 4)));
            if (FORGET) ldsm4(ql, base + M::Q + M::KEY + at<KB>(mt * 16 + (lane & 15), ks * 2 + (lane >> 4)));
#pragma unroll
            for (int np = 0; np < NV / 2; np++) {
                uint32_t bh[4], bl[4];
                ldsm4_t(bh, base + M::S + at<BV>(ks * 16 + (lane & 15), c8 + np * 2 + (lane >> 4)));
                ldsm4_t(bl, base + M::S + M::STATE + at<BV>(ks * 16 + (lane & 15), c8 + np * 2 + (lane >> 4)));
                mma_bf16(o[2 * np], qa, bh[0], bh[1]), mma_bf16(o[2 * np + 1], qa, bh[2], bh[3]);
                mma_bf16(o[2 * np], qa, bl[0], bl[1]), mma_bf16(o[2 * np + 1], qa, bl[2], bl[3]);
                if (FORGET) mma_bf16(o[2 * np], ql, bh[0], bh[1]), mma_bf16(o[2 * np + 1], ql, bh[2], bh[3]);
            }
            if (MLSTM && warp < 4) {
                const float2 n0 = *reinterpret_cast<const float2*>(norm + ks * 16 + 2 * tig), n1 = *reinterpret_cast<const float2*>(norm + ks * 16 + 8 + 2 * tig);
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const uint32_t x = qa[h], y = qa[2 + h];
                    share[h] = fmaf(__uint_as_float(x << 16), n0.x, fmaf(__uint_as_float(x & 0xFFFF0000u), n0.y, share[h]));
                    share[h] = fmaf(__uint_as_float(y << 16), n1.x, fmaf(__uint_as_float(y & 0xFFFF0000u), n1.y, share[h]));
                }
            }
        }
        if (FORGET) {
#pragma unroll
            for (int i = 0; i < NV; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) o[i][j] *= 1.f / E_ONE;
        } else {
            const float f0 = ex2(ea[ta]), f1 = ex2(ea[tb]);
#pragma unroll
            for (int i = 0; i < NV; i++) o[i][0] *= f0, o[i][1] *= f0, o[i][2] *= f1, o[i][3] *= f1;
            if (MLSTM && warp < 4) {
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    share[h] += __shfl_xor_sync(0xffffffffu, share[h], 1);
                    share[h] += __shfl_xor_sync(0xffffffffu, share[h], 2);
                }
                if (tig == 0) nq[ta * 5 + 4] = share[0] * f0, nq[tb * 5 + 4] = share[1] * f1;
            }
        }
    }
    // ---- queries against keys, weighted, to shared memory: ten tiles at and below the diagonal over eight warps.  rect: FORGET, every key before
    // `from` for the queries at and after it.
    auto store_products = [&](int ra, int c0, const float (&p)[4]) {
        uint32_t h0, l0, h1, l1;
        split(p[0], p[1], h0, l0);
        split(p[2], p[3], h1, l1);
        const uint32_t oa = at<C * 2>(ra, c0 >> 3) + (c0 & 7) * 2, ob = at<C * 2>(ra + 8, c0 >> 3) + (c0 & 7) * 2;
        *reinterpret_cast<uint32_t*>(smem + M::P + oa) = h0;
        *reinterpret_cast<uint32_t*>(smem + M::P + M::PROD + oa) = l0;
        *reinterpret_cast<uint32_t*>(smem + M::P + ob) = h1;
        *reinterpret_cast<uint32_t*>(smem + M::P + M::PROD + ob) = l1;
    };
    auto products = [&](bool rect, int from) {
        float held_p[(10 + NW - 1) / NW][2][4];  // a warp's tiles wait until every warp has read the keys
#pragma unroll
        for (int u = 0; u < (10 + NW - 1) / NW; u++) {
            const int t = warp + NW * u;
            if (t >= 10) break;
            const int ti = t < 1 ? 0 : t < 3 ? 1 : t < 6 ? 2 : 3, j = t - ti * (ti + 1) / 2;
            const int ra = ti * 16 + gid, rb = ra + 8;
            float s0[2][4] = {};
#pragma unroll 4
            for (int kp = 0; kp < KS / 2; kp++) {
                uint32_t q0[4], q1[4], l0[4], l1[4];
                const int qr = ti * 16 + (lane & 15), qc = kp * 4 + (lane >> 4);
                ldsm4(q0, base + M::Q + at<KB>(qr, qc));
                ldsm4(q1, base + M::Q + at<KB>(qr, qc + 2));
                if (FORGET) {
                    ldsm4(l0, base + M::Q + M::KEY + at<KB>(qr, qc));
                    ldsm4(l1, base + M::Q + M::KEY + at<KB>(qr, qc + 2));
                }
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    uint32_t b[4], bl[4];
                    const uint32_t off = at<KB>(j * 16 + i * 8 + (lane & 7), kp * 4 + (lane >> 3));
                    ldsm4(b, base + M::K + off);
                    mma_bf16(s0[i], q0, b[0], b[1]), mma_bf16(s0[i], q1, b[2], b[3]);
                    if (FORGET) {
                        ldsm4(bl, base + M::K + M::KEY + off);
                        mma_bf16(s0[i], q0, bl[0], bl[1]), mma_bf16(s0[i], q1, bl[2], bl[3]);
                        mma_bf16(s0[i], l0, b[0], b[1]), mma_bf16(s0[i], l1, b[2], b[3]);
                    }
                }
            }
            float sum[2] = {0.f, 0.f};
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int c0 = j * 16 + i * 8 + 2 * tig;
#pragma unroll
                for (int x = 0; x < 4; x++) {
                    const int c = c0 + (x & 1), r = x < 2 ? ra : rb;
                    const bool seen = rect ? c < from && r >= from : c <= r;
                    s0[i][x] = seen ? FORGET ? s0[i][x] : s0[i][x] * (ex2(ea[r] + eb[c]) * gain[c]) : 0.f;
                    held_p[u][i][x] = s0[i][x];
                }
                sum[0] += s0[i][0] + s0[i][1], sum[1] += s0[i][2] + s0[i][3];
            }
            if (MLSTM) {
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 1);
                    sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 2);
                }
                if (tig == 0) nq[ra * 5 + j] = sum[0], nq[rb * 5 + j] = sum[1];
            }
        }
        __syncthreads();
#pragma unroll
        for (int u = 0; u < (10 + NW - 1) / NW; u++) {
            const int t = warp + NW * u;
            if (t >= 10) break;
            const int ti = t < 1 ? 0 : t < 3 ? 1 : t < 6 ? 2 : 3, j = t - ti * (ti + 1) / 2;
#pragma unroll
            for (int i = 0; i < 2; i++) store_products(ti * 16 + gid, j * 16 + i * 8 + 2 * tig, held_p[u][i]);
        }
    };
    auto times_values = [&]() {
        for (int j = 0; j <= mt; j++) {
            uint32_t ph[4], pl[4];
            ldsm4(ph, base + M::P + at<C * 2>(mt * 16 + (lane & 15), j * 2 + (lane >> 4)));
            ldsm4(pl, base + M::P + M::PROD + at<C * 2>(mt * 16 + (lane & 15), j * 2 + (lane >> 4)));
#pragma unroll
            for (int np = 0; np < NV / 2; np++) {
                uint32_t b[4];
                ldsm4_t(b, base + M::V + at<BV>(j * 16 + (lane & 15), c8 + np * 2 + (lane >> 4)));
                mma_bf16(o[2 * np], ph, b[0], b[1]), mma_bf16(o[2 * np + 1], ph, b[2], b[3]);
                mma_bf16(o[2 * np], pl, b[0], b[1]), mma_bf16(o[2 * np + 1], pl, b[2], b[3]);
            }
        }
    };
    if (!FORGET || !cuts) {
        products(false, 0);
        __syncthreads();
        times_values();
    } else {
        // the chunk is cut: gates and queries come from memory again
        const float2 open = open_of<DK>(a, head, me.ch);
        auto key = [&](int r) {
            if (r >= n || me.ch >= a.dim) return make_float2(0.f, 0.f);
            const float* z = a.gate + (int64_t)(row0 + r) * a.gate_stride + (int64_t)head * a.dim + me.ch;
            return make_float2(one_minus_f(z[0], open.x), one_minus_f(z[1], open.y));
        };
        auto query = [&](int r) {
            if (r >= n || me.ch >= a.dim) return make_float2(0.f, 0.f);
            const __nv_bfloat16* q = gq + r * a.q_stride + me.ch;
            return make_float2(silu(__bfloat162float(q[0])), silu(__bfloat162float(q[1])));
        };
        auto fall = [&](float2& e, int r) {
            const float2 k = key(r);
            e.x *= 1.f - k.x, e.y *= 1.f - k.y;
            return k;
        };
        const int last = me.first + me.TR;
        for (int cut = 0; cut < n;) {
            // where a component of E, counted from the cut, falls too low
            __syncthreads();
            float2 mine = make_float2(1.f, 1.f);
            for (int r = max(cut, me.first); r < last; r++) fall(mine, r);
            me.total(fv, me.part) = mine;
            if (threadIdx.x == 0) cut_end = n;
            __syncthreads();
            float2 e0 = make_float2(E_ONE, E_ONE);
            for (int i = 0; i < me.part; i++) e0.x *= me.total(fv, i).x, e0.y *= me.total(fv, i).y;
            float2 e = e0;
            for (int r = max(cut, me.first); r < min(n, last); r++) {
                fall(e, r);
                if (fminf(e.x, e.y) < E_MIN && r > cut) {
                    atomicMin(&cut_end, r);
                    break;
                }
            }
            __syncthreads();
            const int end = cut_end;
            e = e0;
            for (int r = me.first; r < last; r++) {
                const bool now = r >= cut && r < end;
                float2 k = make_float2(0.f, 0.f), q = k;
                if (now) {
                    k = fall(e, r), q = query(r);
                    e.x = fmaxf(e.x, E_MIN), e.y = fmaxf(e.y, E_MIN);  // a cut's first row may fall further: nothing of the rows before is left then
                }
                put_split(smem + M::Q, smem + M::Q + M::KEY, me.key(r), q.x * e.x, q.y * e.y);
                put_split(smem + M::K, smem + M::K + M::KEY, me.key(r), now ? __fdividef(k.x, e.x) : 0.f, now ? __fdividef(k.y, e.y) : 0.f);
            }
            __syncthreads();
            products(false, 0);
            __syncthreads();
            times_values();
            if (cut > 0) {
                // the rows before the cut: keys brought to it, times the f of the rows between
                __syncthreads();
                mine = make_float2(1.f, 1.f);
                for (int r = me.first; r < min(cut, last); r++) fall(mine, r);
                me.total(fv, me.part) = mine;
                __syncthreads();
                e = make_float2(1.f / E_ONE, 1.f / E_ONE);
                for (int i = me.part + 1; i < me.RS; i++) e.x *= me.total(fv, i).x, e.y *= me.total(fv, i).y;
                for (int r = last - 1; r >= me.first; r--) {
                    const float2 at_cut = e;
                    const float2 k = r < cut ? fall(e, r) : make_float2(0.f, 0.f);
                    put_split(smem + M::K, smem + M::K + M::KEY, me.key(r), k.x * at_cut.x, k.y * at_cut.y);
                }
                __syncthreads();
                products(true, cut);
                __syncthreads();
                times_values();
            }
            cut = end;
        }
    }
    float f[2] = {a.q_scale, a.q_scale};
    if (MLSTM) {
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int t = h ? tb : ta;
            float s = nq[t * 5 + 4];
            for (int j = 0; j <= mt; j++) s += nq[t * 5 + j];
            f[h] = a.q_scale / (fmaxf(fabsf(s * a.q_scale), floor_[t]) + 1e-6f);
        }
    }
    const float skip = SSD ? a.skip[head] : 0.f;
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int t = h ? tb : ta;
        if (t >= n) continue;
        float* dst = a.out + (int64_t)(row0 + t) * a.out_stride + (int64_t)head * a.vdim;
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int c = col0 + (c8 + i) * 8 + 2 * tig;
            float2 v = make_float2(o[i][2 * h] * f[h], o[i][2 * h + 1] * f[h]);
            if (SSD) {
                const uint32_t x = *reinterpret_cast<const uint32_t*>(smem + M::V + at<BV>(t, c8 + i) + tig * 4);
                v.x = fmaf(skip, __uint_as_float(x << 16), v.x), v.y = fmaf(skip, __uint_as_float(x & 0xFFFF0000u), v.y);
            }
            if (c < a.vdim) *reinterpret_cast<float2*>(dst + c) = v;
        }
    }
}

template <int KIND, int DK, int COLS>
cudaError_t launch_add(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RecurrenceChunks& c, const Scratch& s) {
    constexpr size_t smem = AddSmem<KIND, DK, COLS>::BYTES;
    static_assert(smem <= 226 * 1024, "");
    static SmemOptIn configured;
    if (cudaError_t e = tsb_opt_in_smem(ctx, chunk_add_kernel<KIND, DK, COLS>, smem, configured); e != cudaSuccess) return e;
    return tsb_launch(ctx, chunk_add_kernel<KIND, DK, COLS>, dim3((unsigned)((r.vdim + COLS - 1) / COLS), (unsigned)r.heads, (unsigned)c.chunks.n), dim3(THREADS), smem, st,
                      true, r, c.chunks, s, ctx->dev_error);
}
template <int KIND, int DK, int COLS, int NT>
cudaError_t launch_out(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RecurrenceChunks& c, const Scratch& s) {
    constexpr size_t smem = OutSmem<KIND, DK, COLS, NT>::BYTES;
    static_assert(smem <= 226 * 1024, "");
    static SmemOptIn configured;
    if (cudaError_t e = tsb_opt_in_smem(ctx, chunk_out_kernel<KIND, DK, COLS, NT>, smem, configured); e != cudaSuccess) return e;
    return tsb_launch(ctx, chunk_out_kernel<KIND, DK, COLS, NT>, dim3((unsigned)((r.vdim + COLS - 1) / COLS), (unsigned)r.heads, (unsigned)c.chunks.n), dim3(NT), smem, st,
                      true, r, c.chunks, s, ctx->dev_error);
}
template <int KIND, int DK>
cudaError_t launch_chunks(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RecurrenceChunks& c) {
    const Scratch s = scratch_of(r, c.scratch, c.chunks.n);
    cudaError_t e = r.vdim > 64 ? launch_add<KIND, DK, 128>(ctx, st, r, c, s) : launch_add<KIND, DK, 64>(ctx, st, r, c, s);
    const int items = r.dim * r.vdim / 4 + (KIND == REC_MLSTM ? r.dim : 0);
    if (e == cudaSuccess)
        e = tsb_launch(ctx, chunk_walk_kernel<KIND>, dim3((unsigned)((items + THREADS - 1) / THREADS), (unsigned)r.heads, (unsigned)c.n_portions), dim3(THREADS), 0, st, true,
                       r, c, s, ctx->dev_error);
    if (e != cudaSuccess) return e;
    if constexpr (KIND == REC_FORGET)  // the work on queries and keys is the larger part: all value columns share it
        if (r.vdim > 64) return launch_out<KIND, DK, 128, 512>(ctx, st, r, c, s);
    return launch_out<KIND, DK, 64, 256>(ctx, st, r, c, s);
}
template <int KIND>
cudaError_t launch_chunks_dim(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RecurrenceChunks& c) {
    if (r.dim <= 64) return launch_chunks<KIND, 64>(ctx, st, r, c);
    if constexpr (KIND != REC_FORGET)
        if (r.dim > 128) return launch_chunks<KIND, 256>(ctx, st, r, c);
    return launch_chunks<KIND, 128>(ctx, st, r, c);
}

}  // namespace

bool recurrence_chunks_supported(int kind, int dim, int vdim) { return dim <= (kind == REC_FORGET ? 128 : 256) && dim % 8 == 0 && vdim % 8 == 0; }

size_t recurrence_scratch_bytes(int kind, int heads, int dim, int vdim, int chunks) {
    if (!recurrence_chunks_supported(kind, dim, vdim)) return 0;
    const size_t n = (size_t)chunks * heads;
    return align16(n * dim * vdim * 4) + align16(kind == REC_MLSTM ? n * dim * 4 : 0) + align16(n * decay_width(kind, dim) * 4) + align16(n * 8) + (kind == REC_FORGET ? 0 : n * 32 * sizeof(float4));
}

cudaError_t launch_recurrence_chunks(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RecurrenceChunks& c) {
    if (c.chunks.n == 0) return cudaSuccess;
    switch (r.kind) {
        case REC_FORGET: return launch_chunks_dim<REC_FORGET>(ctx, st, r, c);
        case REC_MLSTM: return launch_chunks_dim<REC_MLSTM>(ctx, st, r, c);
        case REC_SSD: return launch_chunks_dim<REC_SSD>(ctx, st, r, c);
        default: return cudaErrorInvalidValue;
    }
}
