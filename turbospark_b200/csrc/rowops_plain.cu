// Row operators of the plain-weight decoders (rowops_plain.cuh).
#include <cuda_bf16.h>

#include <algorithm>
#include <type_traits>

#include "rowops_plain.cuh"

namespace {

constexpr int ROW_THREADS = 256;

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float get(const float* p) { return *p; }
__device__ __forceinline__ float get(const __nv_bfloat16* p) { return __bfloat162float(*p); }

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
    plain_embed_kernel(const T* __restrict__ table, int vocab, int d, const int32_t* tokens, int token_stride, float scale, float* x, T* out,
                       int64_t out_stride, uint32_t* __restrict__ err) {
    pdl_wait();
    pdl_launch_dependents();
    const int tok = tokens[(int64_t)blockIdx.x * token_stride];
    const bool ok = tok >= 0 && tok < vocab;
    if (!ok && threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) {
        const float v = ok ? scale * get(table + (int64_t)tok * d + i) : 0.f;
        x[(int64_t)blockIdx.x * d + i] = v;
        if (out) put(out + (int64_t)blockIdx.x * out_stride + i, v);
    }
}

// sums of squares of one or two rows over the CTA, in a fixed order
__device__ __forceinline__ float2 block_sum2(float2 v) {
    __shared__ float2 red[ROW_THREADS / 32];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        v.x += __shfl_xor_sync(0xffffffffu, v.x, o);
        v.y += __shfl_xor_sync(0xffffffffu, v.y, o);
    }
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float2 t = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < ROW_THREADS / 32; i++) t.x += red[i].x, t.y += red[i].y;
    return t;
}

__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ float sum4(float4 v, float s) { return fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, fmaf(v.x, v.x, s)))); }
__device__ __forceinline__ float mix1(float h, float hp, float mu) { return fmaf(hp - h, mu, h); }

// VEC: d is a multiple of four and at most 4 * ROW_THREADS * ROW_VECS; a thread then holds its columns of both rows in
// registers and everything is read once.
constexpr int ROW_VECS = 4;
template <typename T, bool VEC>
__global__ void __launch_bounds__(ROW_THREADS)
    norm_shift_kernel(const float* x, int d, const float* __restrict__ gain, float eps, const float* __restrict__ mu, const tsb_row_desc* __restrict__ rows,
                      int n_rows, ShiftState state, int layer, int use_before, T* mix_out, T* h_out, int64_t out_stride, uint32_t* __restrict__ err) {
    const int r = blockIdx.x, mask = state.ring_rows - 1;
    // descriptors, gain and the shift's coefficients were written before the pass began
    const tsb_row_desc rd = rows[r];
    const float g = *gain;
    const float* xr = x + (int64_t)r * d;
    const bool in_pass = mu && rd.slot > 0;  // the row before belongs to this pass
    float* keep = nullptr;
    const float* prev = nullptr;
    bool ok = true;
    if (mu) {
        ok = rd.seq >= 0 && rd.seq < state.n_streams;
        if (ok) {
            const int64_t stream = (int64_t)layer * state.n_streams + rd.seq;
            float* ring = state.ring + stream * state.ring_rows * d;
            const int pos = rd.base + rd.slot;
            // the last ring - 1 rows of every portion stay in the state (a stream's rows are consecutive)
            if (r + mask >= n_rows || rows[r + mask].seq != rd.seq) keep = ring + (int64_t)(pos & mask) * d;
            if (!in_pass && pos > 0) prev = use_before ? state.before + stream * d : ring + (int64_t)((pos - 1) & mask) * d;
        }
    }
    float4 m4[VEC ? ROW_VECS : 1];
    if (VEC && mu) {
#pragma unroll
        for (int k = 0; k < ROW_VECS; k++) {
            const int i = (k * ROW_THREADS + threadIdx.x) * 4;
            if (i < d) m4[k] = *reinterpret_cast<const float4*>(mu + i);
        }
    }
    pdl_wait();
    pdl_launch_dependents();
    if (!ok) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        return;
    }
    float2 ss = make_float2(0.f, 0.f);
    if (VEC) {
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        float4 v[ROW_VECS], u[ROW_VECS];
        const float* before = in_pass ? xr - d : prev;
#pragma unroll
        for (int k = 0; k < ROW_VECS; k++) {
            const int i = (k * ROW_THREADS + threadIdx.x) * 4;
            v[k] = i < d ? *reinterpret_cast<const float4*>(xr + i) : zero;
            u[k] = i < d && before ? *reinterpret_cast<const float4*>(before + i) : zero;
        }
#pragma unroll
        for (int k = 0; k < ROW_VECS; k++) ss.x = sum4(v[k], ss.x), ss.y = sum4(u[k], ss.y);
        ss = block_sum2(ss);
        const float s = g / sqrtf(ss.x / (float)d + eps);
        const float sp = in_pass ? g / sqrtf(ss.y / (float)d + eps) : 1.f;  // the state holds normed rows
#pragma unroll
        for (int k = 0; k < ROW_VECS; k++) {
            const int i = (k * ROW_THREADS + threadIdx.x) * 4;
            if (i >= d) break;
            const float4 h = make_float4(v[k].x * s, v[k].y * s, v[k].z * s, v[k].w * s);
            float4 m = h;
            if (mu) {
                m = make_float4(mix1(h.x, u[k].x * sp, m4[k].x), mix1(h.y, u[k].y * sp, m4[k].y), mix1(h.z, u[k].z * sp, m4[k].z),
                                mix1(h.w, u[k].w * sp, m4[k].w));
                if (keep) put4(keep + i, h);
            }
            put4(mix_out + (int64_t)r * out_stride + i, m);
            if (h_out) put4(h_out + (int64_t)r * out_stride + i, h);
        }
        return;
    }
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) {
        const float v = xr[i];
        ss.x = fmaf(v, v, ss.x);
        if (in_pass) {
            const float u = xr[i - d];
            ss.y = fmaf(u, u, ss.y);
        }
    }
    ss = block_sum2(ss);
    const float s = g / sqrtf(ss.x / (float)d + eps), s_prev = g / sqrtf(ss.y / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) {
        const float h = xr[i] * s;
        float m = h;
        if (mu) {
            m = mix1(h, in_pass ? xr[i - d] * s_prev : prev ? prev[i] : 0.f, mu[i]);
            if (keep) keep[i] = h;
        }
        put(mix_out + (int64_t)r * out_stride + i, m);
        if (h_out) put(h_out + (int64_t)r * out_stride + i, h);
    }
}

__global__ void __launch_bounds__(ROW_THREADS) shift_before_kernel(ShiftState state, const tsb_row_desc* __restrict__ rows) {
    pdl_wait();
    pdl_launch_dependents();
    const tsb_row_desc rd = rows[blockIdx.x];
    if (rd.slot != 0 || rd.base <= 0 || rd.seq < 0 || rd.seq >= state.n_streams) return;
    const int64_t stream = (int64_t)blockIdx.y * state.n_streams + rd.seq;
    const float* src = state.ring + (stream * state.ring_rows + ((rd.base - 1) & (state.ring_rows - 1))) * state.width;
    for (int i = threadIdx.x; i < state.width; i += ROW_THREADS) state.before[stream * state.width + i] = src[i];
}

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
    norm_rows_kernel(const float* x, int d, const float* __restrict__ gain, const float* __restrict__ weight, float eps, const int32_t* __restrict__ want,
                     int want_first, int want_step, T* out, int64_t out_stride) {
    pdl_wait();
    pdl_launch_dependents();
    const int r = want ? want[blockIdx.x] : (int)blockIdx.x * want_step + want_first;
    const float* xr = x + (int64_t)r * d;
    float2 ss = make_float2(0.f, 0.f);
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) ss.x = fmaf(xr[i], xr[i], ss.x);
    ss = block_sum2(ss);
    const float s = (weight ? 1.f : *gain) / sqrtf(ss.x / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) put(out + (int64_t)blockIdx.x * out_stride + i, xr[i] * s * (weight ? weight[i] : 1.f));
}

// VEC as in the norm + shift kernel: a thread holds its columns of the row in registers.
template <typename T, bool VEC>
__global__ void __launch_bounds__(ROW_THREADS)
    post_norm_kernel(const float* x, float* x_out, int d, const float* __restrict__ weight, float eps, T* out, int64_t out_stride) {
    const float* xr = x + (int64_t)blockIdx.x * d;
    float* xo = x_out ? x_out + (int64_t)blockIdx.x * d : nullptr;  // may be the row itself
    T* o = out + (int64_t)blockIdx.x * out_stride;
    float4 w[VEC ? ROW_VECS : 1];
    if (VEC) {
#pragma unroll
        for (int k = 0; k < ROW_VECS; k++) {
            const int i = (k * ROW_THREADS + threadIdx.x) * 4;
            if (i < d) w[k] = *reinterpret_cast<const float4*>(weight + i);
        }
    }
    pdl_wait();
    pdl_launch_dependents();
    float2 ss = make_float2(0.f, 0.f);
    if (VEC) {
        float4 v[ROW_VECS];
#pragma unroll
        for (int k = 0; k < ROW_VECS; k++) {
            const int i = (k * ROW_THREADS + threadIdx.x) * 4;
            v[k] = i < d ? *reinterpret_cast<const float4*>(xr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int k = 0; k < ROW_VECS; k++) ss.x = sum4(v[k], ss.x);
        const float s = 1.f / sqrtf(block_sum2(ss).x / (float)d + eps);
#pragma unroll
        for (int k = 0; k < ROW_VECS; k++) {
            const int i = (k * ROW_THREADS + threadIdx.x) * 4;
            if (i >= d) break;
            const float4 h = make_float4(v[k].x * s * w[k].x, v[k].y * s * w[k].y, v[k].z * s * w[k].z, v[k].w * s * w[k].w);
            if (xo) put4(xo + i, h);
            put4(o + i, h);
        }
        return;
    }
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) ss.x = fmaf(xr[i], xr[i], ss.x);
    const float s = 1.f / sqrtf(block_sum2(ss).x / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) {
        const float h = xr[i] * s * weight[i];
        if (xo) xo[i] = h;
        put(o + i, h);
    }
}

// Columns c .. of a block's mean: the cache's rows at its positions, summed in their order, eight loads in flight.
template <typename T>
__device__ __forceinline__ void block_mean(const KeyView& keys, int pool, int seq, int block, int c, T* dst) {
    constexpr int N = 16 / sizeof(T), AHEAD = 8;
    float sum[N];
#pragma unroll
    for (int i = 0; i < N; i++) sum[i] = 0.f;
    for (int j0 = 0; j0 < pool; j0 += AHEAD) {
        const T* src[AHEAD];
        uint4 v[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; j++) src[j] = j0 + j < pool ? key_row<T>(keys, seq, block * pool + j0 + j) : nullptr;  // reserved, as later ones are
#pragma unroll
        for (int j = 0; j < AHEAD; j++) v[j] = src[j] ? *reinterpret_cast<const uint4*>(src[j] + c) : make_uint4(0, 0, 0, 0);
#pragma unroll
        for (int j = 0; j < AHEAD; j++) {
            const T* e = reinterpret_cast<const T*>(&v[j]);
#pragma unroll
            for (int i = 0; i < N; i++) sum[i] += get(e + i);
        }
    }
#pragma unroll
    for (int i = 0; i < N; i++) put(dst + c + i, sum[i] / (float)pool);
}

// the pair of columns i and i + 1 (i even), turned; columns behind the turned ones pass
__device__ __forceinline__ void turn_pair(const float2* table, int half, int r, int i, float& u, float& v) {
    if (i >= 2 * half) return;
    const float2 t = table[(int64_t)r * half + (i >> 1)];
    const float x = fmaf(u, t.x, -v * t.y);
    v = fmaf(v, t.x, u * t.y), u = x;
}

// LANES lanes per (row, head).  VEC > 0: the width is a multiple of four and at most 4 LANES VEC, and a lane holds its columns in
// registers.
template <typename T, int LANES, int VEC, bool MORE>
__global__ void __launch_bounds__(ROW_THREADS) head_norms_kernel(const __grid_constant__ HeadNorms h, int rows, uint32_t* __restrict__ err) {
    const int lane = threadIdx.x & (LANES - 1);
    const int64_t item = (int64_t)blockIdx.x * (ROW_THREADS / LANES) + threadIdx.x / LANES;
    const int per = h.n_q + h.n_k + (MORE ? h.n_v + (h.pool > 0 ? h.keys.kv_heads : 0) : 0);
    const bool in = item < (int64_t)rows * per;
    const int r = in ? (int)(item / per) : 0, head = in ? (int)(item % per) : 0;
    const tsb_row_desc rd = h.rows[r];
    pdl_wait();
    pdl_launch_dependents();
    if (!in) return;
    const bool query = head < h.n_q, value = MORE && head >= h.n_q + h.n_k;
    if (MORE && head >= h.n_q + h.n_k + h.n_v) {
        const int pos = rd.base + rd.slot, block = pos / h.pool - 1, at = (head - h.n_q - h.n_k - h.n_v) * h.keys.head_step;
        if (rd.slot != 0 || block < 0 || (block + 1) * h.pool != pos) return;
        T* dst = key_row<T>(h.pooled, rd.seq, block);
        if (!dst && lane == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        for (int c = lane * (16 / (int)sizeof(T)); dst && c < h.keys.head_step; c += LANES * (16 / (int)sizeof(T))) block_mean<T>(h.keys, h.pool, rd.seq, block, at + c, dst);
        return;
    }
    const float* src = h.raw + (int64_t)r * h.raw_stride + (int64_t)head * h.width;
    if (value) {
        src += (int64_t)(head - h.n_q - h.n_k) * (h.v_width - h.width);
        T* dst = key_row<T>(h.keys, rd.seq, rd.base + rd.slot);
        if (!dst) {
            if (lane == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
            return;
        }
        dst += (int64_t)(head - h.n_q - h.n_k) * h.keys.head_step + h.keys.value_off;
        if (VEC > 0) {
#pragma unroll
            for (int k = 0; k < VEC; k++) {
                const int i = (k * LANES + lane) * 4;
                if (i >= h.v_width) break;
                float4 v = *reinterpret_cast<const float4*>(src + i);
                turn_pair(h.turn, h.turn_half, r, i, v.x, v.y), turn_pair(h.turn, h.turn_half, r, i + 2, v.z, v.w);
                put4(dst + i, v);
            }
            return;
        }
        for (int i = 2 * lane; i < h.v_width; i += 2 * LANES) {
            float u = src[i], v = i + 1 < h.v_width ? src[i + 1] : 0.f;
            turn_pair(h.turn, h.turn_half, r, i, u, v);
            put(dst + i, u);
            if (i + 1 < h.v_width) put(dst + i + 1, v);
        }
        return;
    }
    const float* w = query ? h.q_weight : h.k_weight;
    float ss = 0.f;
    float4 v[VEC > 0 ? VEC : 1], g[VEC > 0 ? VEC : 1];
    if (VEC > 0) {
#pragma unroll
        for (int k = 0; k < VEC; k++) {
            const int i = (k * LANES + lane) * 4;
            v[k] = i < h.width ? *reinterpret_cast<const float4*>(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            g[k] = i < h.width ? *reinterpret_cast<const float4*>(w + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int k = 0; k < VEC; k++) ss = sum4(v[k], ss);
    } else {
        for (int i = lane; i < h.width; i += LANES) ss = fmaf(src[i], src[i], ss);
    }
    const uint32_t mask = LANES == 32 ? 0xffffffffu : ((1u << (LANES & 31)) - 1) << (threadIdx.x & 31 & ~(LANES - 1));
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
    float s = 1.f / sqrtf(ss / (float)h.width + h.eps);
    const int pos = rd.base + rd.slot;
    T* dst;
    int width = h.width;
    if (query) {
        if (h.temp_every > 0) s *= 1.f + h.temp_coef * logf((float)((pos + 1) / h.temp_every + 1));
        dst = static_cast<T*>(h.q) + (int64_t)r * h.q_stride + (int64_t)head * h.q_step;
        width = h.q_width;
    } else {
        dst = key_row<T>(h.keys, rd.seq, pos);
        if (!dst) {
            if (lane == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
            return;
        }
        dst += (int64_t)(head - h.n_q) * h.keys.head_step;
    }
    if (VEC > 0) {
#pragma unroll
        for (int k = 0; k < VEC; k++) {
            const int i = (k * LANES + lane) * 4;
            if (i >= h.width) break;
            float4 o = make_float4(v[k].x * s * g[k].x, v[k].y * s * g[k].y, v[k].z * s * g[k].z, v[k].w * s * g[k].w);
            if (MORE && h.rot) turn_pair(h.rot, h.rot_half, r, i, o.x, o.y), turn_pair(h.rot, h.rot_half, r, i + 2, o.z, o.w);
            put4(dst + i, o);
        }
        for (int i = h.width + lane; i < width; i += LANES) put(dst + i, 0.f);
        return;
    }
    for (int i = 2 * lane; i < width; i += 2 * LANES) {
        float u = i < h.width ? src[i] * s * w[i] : 0.f, v = i + 1 < h.width ? src[i + 1] * s * w[i + 1] : 0.f;
        if (MORE && h.rot) turn_pair(h.rot, h.rot_half, r, i, u, v);
        put(dst + i, u);
        if (i + 1 < width) put(dst + i + 1, v);
    }
}

__global__ void __launch_bounds__(ROW_THREADS)
    rotary_table_kernel(const double* __restrict__ freq, int half, float magnitude, const tsb_row_desc* __restrict__ rows, int n, float2* table) {
    pdl_wait();
    pdl_launch_dependents();
    const int64_t k = (int64_t)blockIdx.x * ROW_THREADS + threadIdx.x;
    if (k >= (int64_t)n * half) return;
    const tsb_row_desc& rd = rows[k / half];
    constexpr double TURN = 6.283185307179586476925;
    double a = (double)(rd.base + rd.slot) * freq[k % half];
    a -= TURN * rint(a * (1.0 / TURN));
    float s, c;
    sincosf((float)a, &s, &c);
    table[k] = make_float2(magnitude * c, magnitude * s);
}

// Rows that end no block leave at once; a thread sums eight (f32: four) columns.
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS) block_means_kernel(const __grid_constant__ BlockMeans b, uint32_t* __restrict__ err) {
    constexpr int N = 16 / sizeof(T);
    const tsb_row_desc rd = b.rows[blockIdx.x];
    const int pos = rd.base + rd.slot, block = pos / b.pool;
    pdl_wait();
    pdl_launch_dependents();
    if (pos - block * b.pool != b.pool - 1) return;
    T* dst = key_row<T>(b.pooled, rd.seq, block);
    if (!dst) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        return;
    }
    for (int c = threadIdx.x * N; c < b.keys.row; c += ROW_THREADS * N) block_mean<T>(b.keys, b.pool, rd.seq, block, c, dst);
}

// a CTA per position and stream
__global__ void __launch_bounds__(ROW_THREADS) latent_gather_kernel(const __grid_constant__ LatentGather g, uint32_t* __restrict__ err) {
    const ExpandStream es = g.streams[blockIdx.y];
    const tsb_row_desc rd = g.rows[es.first_row];
    const int pos = blockIdx.x, len = rd.base + es.n_rows;
    pdl_wait();
    pdl_launch_dependents();
    if (pos >= len) return;
    const int wide_lp = pos >> g.wide.page_shift, wide_page = es.first_page + wide_lp;
    if (rd.seq < 0 || rd.seq >= g.wide.max_seqs || wide_lp >= g.wide.max_pages_per_seq || wide_page >= g.wide.num_pages) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        return;
    }
    if (threadIdx.x == 0 && (pos & (g.wide.page_tokens - 1)) == 0) g.wide_table[(int64_t)rd.seq * g.wide.max_pages_per_seq + wide_lp] = wide_page;
    const __nv_bfloat16* src = key_row<__nv_bfloat16>(g.cache, rd.seq, pos);
    if (!src) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        return;
    }
    const int64_t at = (int64_t)wide_page * g.wide.page_tokens + (pos & (g.wide.page_tokens - 1));
    const uint4* s16 = reinterpret_cast<const uint4*>(src);
    uint4* d16 = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(g.latents) + at * g.cache.row);
    for (int i = threadIdx.x; i < g.cache.row / 8; i += ROW_THREADS) d16[i] = s16[i];
    __nv_bfloat16* wide = reinterpret_cast<__nv_bfloat16*>(g.wide.base) + at * g.wide.row;
    const int tail = g.wide.head_dim - g.key_off;
    for (int i = threadIdx.x; i < g.wide.kv_heads * tail; i += ROW_THREADS) {
        const int head = i / tail, k = i - head * tail;
        wide[(int64_t)head * g.wide.head_step + g.key_off + k] = k < g.rot_dim ? src[g.kv_rank + k] : __float2bfloat16_rn(0.f);
    }
}

}  // namespace

cudaError_t launch_plain_embed(tsb_ctx* ctx, cudaStream_t st, bool f32, const void* table, int vocab, int d, const int32_t* tokens, int token_stride,
                               int rows, float scale, float* x, void* out, int64_t out_stride) {
    if (f32)
        return tsb_launch(ctx, plain_embed_kernel<float>, dim3((unsigned)rows), dim3(ROW_THREADS), 0, st, true, (const float*)table, vocab, d, tokens,
                          token_stride, scale, x, (float*)out, out_stride, ctx->dev_error);
    return tsb_launch(ctx, plain_embed_kernel<__nv_bfloat16>, dim3((unsigned)rows), dim3(ROW_THREADS), 0, st, true, (const __nv_bfloat16*)table, vocab, d,
                      tokens, token_stride, scale, x, (__nv_bfloat16*)out, out_stride, ctx->dev_error);
}

cudaError_t launch_norm_shift(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* gain, float eps, const float* mu,
                              const tsb_row_desc* rows_dev, int rows, ShiftState state, int layer, bool use_before, void* mix_out, void* h_out,
                              int64_t out_stride) {
    auto run = [&](auto kernel, auto* mix, auto* h) {
        return tsb_launch(ctx, kernel, dim3((unsigned)rows), dim3(ROW_THREADS), 0, st, true, x, d, gain, eps, mu, rows_dev, rows, state, layer,
                          (int)use_before, mix, h, out_stride, ctx->dev_error);
    };
    const bool vec = d % 4 == 0 && out_stride % 4 == 0 && d <= 4 * ROW_THREADS * ROW_VECS;
    if (f32) return run(vec ? norm_shift_kernel<float, true> : norm_shift_kernel<float, false>, (float*)mix_out, (float*)h_out);
    return run(vec ? norm_shift_kernel<__nv_bfloat16, true> : norm_shift_kernel<__nv_bfloat16, false>, (__nv_bfloat16*)mix_out, (__nv_bfloat16*)h_out);
}

cudaError_t launch_shift_before(tsb_ctx* ctx, cudaStream_t st, ShiftState state, int layers, const tsb_row_desc* rows_dev, int rows) {
    return tsb_launch(ctx, shift_before_kernel, dim3((unsigned)rows, (unsigned)layers), dim3(ROW_THREADS), 0, st, true, state, rows_dev);
}

cudaError_t launch_norm_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* gain, const float* weight, float eps,
                             const int32_t* want_dev, int want_first, int want_step, int n, void* out, int64_t out_stride) {
    if (f32)
        return tsb_launch(ctx, norm_rows_kernel<float>, dim3((unsigned)n), dim3(ROW_THREADS), 0, st, true, x, d, gain, weight, eps, want_dev, want_first,
                          want_step, (float*)out, out_stride);
    return tsb_launch(ctx, norm_rows_kernel<__nv_bfloat16>, dim3((unsigned)n), dim3(ROW_THREADS), 0, st, true, x, d, gain, weight, eps, want_dev,
                      want_first, want_step, (__nv_bfloat16*)out, out_stride);
}

static cudaError_t launch_norm_of(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, float* x_out, int d, const float* weight, float eps, int rows, void* out,
                                  int64_t out_stride) {
    auto run = [&](auto kernel, auto* o) {
        return tsb_launch(ctx, kernel, dim3((unsigned)rows), dim3(ROW_THREADS), 0, st, true, x, x_out, d, weight, eps, o, out_stride);
    };
    const bool vec = d % 4 == 0 && out_stride % 4 == 0 && d <= 4 * ROW_THREADS * ROW_VECS;
    if (f32) return run(vec ? post_norm_kernel<float, true> : post_norm_kernel<float, false>, (float*)out);
    return run(vec ? post_norm_kernel<__nv_bfloat16, true> : post_norm_kernel<__nv_bfloat16, false>, (__nv_bfloat16*)out);
}
cudaError_t launch_post_norm(tsb_ctx* ctx, cudaStream_t st, bool f32, float* x, int d, const float* weight, float eps, int rows, void* out,
                             int64_t out_stride) {
    return launch_norm_of(ctx, st, f32, x, x, d, weight, eps, rows, out, out_stride);
}
cudaError_t launch_pre_norm(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* weight, float eps, int rows, void* out,
                            int64_t out_stride) {
    return launch_norm_of(ctx, st, f32, x, nullptr, d, weight, eps, rows, out, out_stride);
}

cudaError_t launch_head_norms(tsb_ctx* ctx, cudaStream_t st, bool f32, const HeadNorms& h, int rows) {
    auto run = [&](auto kernel, int lanes) {
        const int per_cta = ROW_THREADS / lanes;
        const dim3 grid((unsigned)(((int64_t)rows * (h.n_q + h.n_k + h.n_v + (h.pool > 0 ? h.keys.kv_heads : 0)) + per_cta - 1) / per_cta));
        return tsb_launch(ctx, kernel, grid, dim3(ROW_THREADS), 0, st, true, h, rows, ctx->dev_error);
    };
    const int wide = h.n_v > 0 ? std::max(h.width, h.v_width) : h.width;
    const bool vec = h.width % 4 == 0 && (h.n_v == 0 || h.v_width % 4 == 0) && wide <= 512 && h.raw_stride % 4 == 0 && (uintptr_t)h.raw % 16 == 0 && h.q_step % 4 == 0 && h.q_stride % 4 == 0;
    // MORE: rotations, values, blocks
    const bool more = h.rot || h.n_v > 0 || h.pool > 0;
    auto pick = [&](auto type, auto with) {
        using T = decltype(type);
        constexpr bool MORE = decltype(with)::value;
        if (vec && wide <= 64) return run(head_norms_kernel<T, 8, 2, MORE>, 8);
        if (vec && wide <= 128) return run(head_norms_kernel<T, 16, 2, MORE>, 16);
        return vec ? run(head_norms_kernel<T, 32, 4, MORE>, 32) : run(head_norms_kernel<T, 32, 0, MORE>, 32);
    };
    if (f32) return more ? pick(0.f, std::true_type{}) : pick(0.f, std::false_type{});
    return more ? pick(__nv_bfloat16{}, std::true_type{}) : pick(__nv_bfloat16{}, std::false_type{});
}

cudaError_t launch_block_means(tsb_ctx* ctx, cudaStream_t st, bool f32, const BlockMeans& b, int rows) {
    auto run = [&](auto kernel) { return tsb_launch(ctx, kernel, dim3((unsigned)rows), dim3(ROW_THREADS), 0, st, true, b, ctx->dev_error); };
    return f32 ? run(block_means_kernel<float>) : run(block_means_kernel<__nv_bfloat16>);
}

cudaError_t launch_rotary_table(tsb_ctx* ctx, cudaStream_t st, const double* freq, int half, float magnitude, const tsb_row_desc* rows_dev, int rows,
                                float2* table) {
    return tsb_launch(ctx, rotary_table_kernel, dim3((unsigned)(((int64_t)rows * half + ROW_THREADS - 1) / ROW_THREADS)), dim3(ROW_THREADS), 0, st, true, freq,
                      half, magnitude, rows_dev, rows, table);
}

cudaError_t launch_latent_gather(tsb_ctx* ctx, cudaStream_t st, const LatentGather& g, int n_streams, int max_len) {
    return tsb_launch(ctx, latent_gather_kernel, dim3((unsigned)max_len, (unsigned)n_streams), dim3(ROW_THREADS), 0, st, true, g, ctx->dev_error);
}
