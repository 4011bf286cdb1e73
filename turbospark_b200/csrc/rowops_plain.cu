// Row operators of the plain-weight decoders (rowops_plain.cuh).
#include <cuda_bf16.h>

#include "rowops_plain.cuh"

namespace {

constexpr int ROW_THREADS = 256;

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float get(const float* p) { return *p; }
__device__ __forceinline__ float get(const __nv_bfloat16* p) { return __bfloat162float(*p); }

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
    plain_embed_kernel(const T* __restrict__ table, int vocab, int d, const int32_t* tokens, int token_stride, float* x, uint32_t* __restrict__ err) {
    pdl_wait();
    pdl_launch_dependents();
    const int tok = tokens[(int64_t)blockIdx.x * token_stride];
    const bool ok = tok >= 0 && tok < vocab;
    if (!ok && threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) x[(int64_t)blockIdx.x * d + i] = ok ? get(table + (int64_t)tok * d + i) : 0.f;
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
    norm_rows_kernel(const float* x, int d, const float* __restrict__ gain, float eps, const int32_t* __restrict__ want, int want_first, int want_step,
                     T* out, int64_t out_stride) {
    pdl_wait();
    pdl_launch_dependents();
    const int r = want ? want[blockIdx.x] : (int)blockIdx.x * want_step + want_first;
    const float* xr = x + (int64_t)r * d;
    float2 ss = make_float2(0.f, 0.f);
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) ss.x = fmaf(xr[i], xr[i], ss.x);
    ss = block_sum2(ss);
    const float s = *gain / sqrtf(ss.x / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) put(out + (int64_t)blockIdx.x * out_stride + i, xr[i] * s);
}

}  // namespace

cudaError_t launch_plain_embed(tsb_ctx* ctx, cudaStream_t st, bool f32, const void* table, int vocab, int d, const int32_t* tokens, int token_stride,
                               int rows, float* x) {
    if (f32)
        return tsb_launch(ctx, plain_embed_kernel<float>, dim3((unsigned)rows), dim3(ROW_THREADS), 0, st, true, (const float*)table, vocab, d, tokens,
                          token_stride, x, ctx->dev_error);
    return tsb_launch(ctx, plain_embed_kernel<__nv_bfloat16>, dim3((unsigned)rows), dim3(ROW_THREADS), 0, st, true, (const __nv_bfloat16*)table, vocab, d,
                      tokens, token_stride, x, ctx->dev_error);
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

cudaError_t launch_norm_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* gain, float eps, const int32_t* want_dev,
                             int want_first, int want_step, int n, void* out, int64_t out_stride) {
    if (f32)
        return tsb_launch(ctx, norm_rows_kernel<float>, dim3((unsigned)n), dim3(ROW_THREADS), 0, st, true, x, d, gain, eps, want_dev, want_first, want_step,
                          (float*)out, out_stride);
    return tsb_launch(ctx, norm_rows_kernel<__nv_bfloat16>, dim3((unsigned)n), dim3(ROW_THREADS), 0, st, true, x, d, gain, eps, want_dev, want_first,
                      want_step, (__nv_bfloat16*)out, out_stride);
}
