// Choice of experts and the lists of the grouped products (experts.cuh).
#include "experts.cuh"

namespace {

constexpr int ROUTE_WARPS = 4, LIST_THREADS = 256;

struct Best {
    float v;
    int i;
};
__device__ __forceinline__ Best better(Best a, Best b) { return b.v > a.v || (b.v == a.v && b.i < a.i) ? b : a; }
__device__ __forceinline__ Best warp_best(Best b) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) b = better(b, Best{__shfl_xor_sync(0xffffffffu, b.v, o), __shfl_xor_sync(0xffffffffu, b.i, o)});
    return b;
}

// A warp per row.  Shared memory per warp: choice [experts], worth of the groups [groups].
__global__ void __launch_bounds__(ROUTE_WARPS * 32) route_kernel(const __grid_constant__ ExpertRouting r) {
    extern __shared__ float smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x * ROUTE_WARPS + warp;
    float *choice = smem + warp * (r.experts + r.groups), *worth = choice + r.experts;
    pdl_wait();
    pdl_launch_dependents();
    if (row >= r.rows) return;
    const float* z = r.logits + (int64_t)row * r.logits_stride;
    auto score = [&](int e) { return 1.f / (1.f + expf(-z[e])); };
    for (int e = lane; e < r.experts; e += 32) choice[e] = score(e) + r.correction[e];
    __syncwarp();
    const int per = r.experts / r.groups;
    if (r.keep < r.groups) {
        for (int g = lane; g < r.groups; g += 32) {
            float a = -INFINITY, b = -INFINITY;  // the largest and the second largest
            for (int i = 0; i < per; i++) {
                const float v = choice[g * per + i];
                b = fmaxf(b, fminf(a, v)), a = fmaxf(a, v);
            }
            worth[g] = per > 1 ? a + b : a;
        }
        __syncwarp();
        // the groups that stay get a mark
        for (int k = 0; k < r.keep; k++) {
            Best best{-INFINITY, 0x7fffffff};
            for (int g = lane; g < r.groups; g += 32)
                if (!isnan(worth[g])) best = better(best, Best{worth[g], g});
            best = warp_best(best);
            if (lane == 0 && best.i < r.groups) worth[best.i] = __int_as_float(0x7fc00000);
            __syncwarp();
        }
        for (int e = lane; e < r.experts; e += 32)
            if (!isnan(worth[e / per])) choice[e] = -INFINITY;
        __syncwarp();
    }
    for (int k = 0; k < r.top; k++) {
        Best best{-INFINITY, 0x7fffffff};
        for (int e = lane; e < r.experts; e += 32) best = better(best, Best{choice[e], e});
        best = warp_best(best);
        const int e = min(best.i, r.experts - 1);
        if (lane == 0) {
            r.lists.ids[(int64_t)row * r.top + k] = e, r.lists.weight[(int64_t)row * r.top + k] = score(e);
            choice[e] = -INFINITY;
        }
        __syncwarp();
    }
}

// A CTA per expert: its slots in row order.  Every CTA counts all experts (integers: the order does not matter), so none waits for another.
__global__ void __launch_bounds__(LIST_THREADS) expert_lists_kernel(const __grid_constant__ ExpertRouting r) {
    extern __shared__ int count[];  // [experts]
    __shared__ int red[2][LIST_THREADS / 32];
    const int e = blockIdx.x, n = r.rows * r.top, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int i = threadIdx.x; i < r.experts; i += LIST_THREADS) count[i] = 0;
    __syncthreads();
    pdl_wait();
    pdl_launch_dependents();
    for (int i = threadIdx.x; i < n; i += LIST_THREADS) atomicAdd(&count[r.lists.ids[i]], 1);
    __syncthreads();
    int slots = 0, chunks = 0;  // of the experts before this one
    for (int i = threadIdx.x; i < e; i += LIST_THREADS) slots += count[i], chunks += (count[i] + r.chunk_slots - 1) / r.chunk_slots;
    slots = __reduce_add_sync(0xffffffffu, slots), chunks = __reduce_add_sync(0xffffffffu, chunks);
    if (lane == 0) red[0][warp] = slots, red[1][warp] = chunks;
    __syncthreads();
    slots = chunks = 0;
    for (int i = 0; i < LIST_THREADS / 32; i++) slots += red[0][i], chunks += red[1][i];
    const int mine = count[e], my_chunks = (mine + r.chunk_slots - 1) / r.chunk_slots;
    if (threadIdx.x == 0) {
        r.lists.first[e] = slots;
        if (e == r.experts - 1) r.lists.first[r.experts] = slots + mine, *r.lists.n_chunks = chunks + my_chunks;
    }
    for (int c = threadIdx.x; c < my_chunks; c += LIST_THREADS)
        r.lists.chunks[chunks + c] = ExpertChunk{e, slots + c * r.chunk_slots, min(r.chunk_slots, mine - c * r.chunk_slots)};
    if (mine == 0) return;
    int at = slots;
    for (int i0 = 0; i0 < n; i0 += LIST_THREADS) {
        const int i = i0 + threadIdx.x;
        const bool hit = i < n && r.lists.ids[i] == e;
        const uint32_t hits = __ballot_sync(0xffffffffu, hit);
        __syncthreads();
        if (lane == 0) red[0][warp] = __popc(hits);
        __syncthreads();
        int before = 0, all = 0;
#pragma unroll
        for (int w = 0; w < LIST_THREADS / 32; w++) {
            const int h = red[0][w];
            if (w < warp) before += h;
            all += h;
        }
        if (hit) {
            const int slot = at + before + __popc(hits & ((1u << lane) - 1));
            r.lists.slot_of[i] = slot, r.lists.token_of[slot] = i / r.top;
        }
        at += all;
    }
}

__global__ void __launch_bounds__(256) gather_rows_kernel(const uint8_t* x, int64_t x_bytes, const int32_t* token_of, uint8_t* out, int64_t bytes) {
    pdl_wait();
    pdl_launch_dependents();
    const uint4* src = reinterpret_cast<const uint4*>(x + (int64_t)token_of[blockIdx.x] * x_bytes);
    uint4* dst = reinterpret_cast<uint4*>(out + (int64_t)blockIdx.x * bytes);
    for (int64_t i = threadIdx.x; i < bytes / 16; i += 256) dst[i] = src[i];
}

}  // namespace

bool routing_supported(int experts, int top, int groups, int keep) {
    return experts > 0 && experts <= EXPERTS_MAX && groups > 0 && experts % groups == 0 && keep > 0 && keep <= groups && top > 0 && top <= experts / groups * keep;
}

cudaError_t launch_route_experts(tsb_ctx* ctx, cudaStream_t st, const ExpertRouting& r) {
    cudaError_t e = tsb_launch(ctx, route_kernel, dim3((unsigned)((r.rows + ROUTE_WARPS - 1) / ROUTE_WARPS)), dim3(ROUTE_WARPS * 32),
                               (size_t)ROUTE_WARPS * (r.experts + r.groups) * sizeof(float), st, true, r);
    if (e != cudaSuccess) return e;
    return tsb_launch(ctx, expert_lists_kernel, dim3((unsigned)r.experts), dim3(LIST_THREADS), (size_t)r.experts * sizeof(int), st, true, r);
}

cudaError_t launch_gather_rows(tsb_ctx* ctx, cudaStream_t st, const void* x, int64_t x_bytes, const int32_t* token_of, int slots, void* out, int64_t bytes) {
    return tsb_launch(ctx, gather_rows_kernel, dim3((unsigned)slots), dim3(256), 0, st, true, (const uint8_t*)x, x_bytes, token_of, (uint8_t*)out, bytes);
}
