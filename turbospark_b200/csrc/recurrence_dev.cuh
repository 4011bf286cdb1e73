// Gates of the recurrent mixers, shared by the row-by-row and the chunked kernels.  All f32.
#pragma once
#include <cuda_bf16.h>

#include "recurrence.cuh"

namespace {

__device__ __forceinline__ float rec_get(const float* p) { return *p; }
__device__ __forceinline__ float rec_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float rec_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float rec_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float rec_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float rec_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// log input gate and log forget gate of an mLSTM head
__device__ __forceinline__ float2 mlstm_gates(const Recurrence& r, int row, int head) {
    const float* g = r.gate + (int64_t)row * r.gate_stride + head;
    return make_float2(r.cap * tanhf(g[0] / r.cap), rec_log_sigmoid(r.cap * tanhf(g[r.heads] / r.cap)));
}
// step size and log decay of an SSD head; rate = exp(a_log)
__device__ __forceinline__ float2 ssd_gates(const Recurrence& r, int row, int head, float rate) {
    const float dt = rec_softplus(r.gate[(int64_t)row * r.gate_stride + head]);
    return make_float2(dt, -rate * dt);
}

__device__ __forceinline__ int64_t rec_slot(const Recurrence& r, int seq, int pos) { return (int64_t)seq * r.state.ring + (pos & (r.state.ring - 1)); }

}  // namespace
