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

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
    norm_shift_kernel(const float* x, int d, const float* __restrict__ gain, float eps, const float* __restrict__ mu, const tsb_row_desc* __restrict__ rows,
                      int n_rows, ShiftState state, int layer, int use_before, T* mix_out, T* h_out, int64_t out_stride, uint32_t* __restrict__ err) {
    const int r = blockIdx.x;
    pdl_wait();
    pdl_launch_dependents();
    const tsb_row_desc rd = rows[r];
    const float* xr = x + (int64_t)r * d;
    const bool in_pass = mu && rd.slot > 0;  // the row before belongs to this pass
    float2 ss = make_float2(0.f, 0.f);
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) {
        const float v = xr[i];
        ss.x = fmaf(v, v, ss.x);
        if (in_pass) {
            const float u = xr[i - d];
            ss.y = fmaf(u, u, ss.y);
        }
    }
    ss = block_sum2(ss);
    const float g = *gain;
    const float s = g / sqrtf(ss.x / (float)d + eps), s_prev = g / sqrtf(ss.y / (float)d + eps);
    float* keep = nullptr;
    const float* prev = nullptr;
    if (mu) {
        if (rd.seq < 0 || rd.seq >= state.n_streams) {
            if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
            return;
        }
        const int64_t stream = (int64_t)layer * state.n_streams + rd.seq;
        float* ring = state.ring + stream * state.ring_rows * d;
        const int pos = rd.base + rd.slot, mask = state.ring_rows - 1;
        // the last ring - 1 rows of every portion stay in the state (a stream's rows are consecutive)
        if (r + mask >= n_rows || rows[r + mask].seq != rd.seq) keep = ring + (int64_t)(pos & mask) * d;
        if (!in_pass && pos > 0) prev = use_before ? state.before + stream * d : ring + (int64_t)((pos - 1) & mask) * d;
    }
    for (int i = threadIdx.x; i < d; i += ROW_THREADS) {
        const float h = xr[i] * s;
        float m = h;
        if (mu) {
            const float hp = in_pass ? xr[i - d] * s_prev : prev ? prev[i] : 0.f;
            m = fmaf(hp - h, mu[i], h);
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
    if (f32)
        return tsb_launch(ctx, norm_shift_kernel<float>, dim3((unsigned)rows), dim3(ROW_THREADS), 0, st, true, x, d, gain, eps, mu, rows_dev, rows, state,
                          layer, (int)use_before, (float*)mix_out, (float*)h_out, out_stride, ctx->dev_error);
    return tsb_launch(ctx, norm_shift_kernel<__nv_bfloat16>, dim3((unsigned)rows), dim3(ROW_THREADS), 0, st, true, x, d, gain, eps, mu, rows_dev, rows,
                      state, layer, (int)use_before, (__nv_bfloat16*)mix_out, (__nv_bfloat16*)h_out, out_stride, ctx->dev_error);
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
