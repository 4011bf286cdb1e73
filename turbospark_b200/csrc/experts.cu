// Choice of experts and the lists of the grouped products (experts.cuh).
#include <algorithm>

#include "experts.cuh"

namespace {

constexpr int ROUTE_WARPS = 4, LIST_THREADS = 256;
constexpr int RANK_MAX = 128;                      // experts up to which the choice is by rank
constexpr int SMALL_ROWS = 32, SMALL_PAIRS = 512;  // passes whose choice and lists one CTA makes

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

// The choice of one row by one warp.  Shared memory of the warp: choice [experts], worth of the groups [groups], picked [top].
__device__ __forceinline__ void route_row(const ExpertRouting& r, int row, float* choice, int lane) {
    float* worth = choice + r.experts;
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
        // a group stays if fewer than `keep` are better
        for (int e = lane; e < r.experts; e += 32) {
            const int mine = e / per;
            const float w = worth[mine];
            int better_ones = 0;
            for (int g = 0; g < r.groups; g++) better_ones += worth[g] > w || (worth[g] == w && g < mine);
            if (better_ones >= r.keep) choice[e] = -INFINITY;
        }
        __syncwarp();
    }
    int32_t* ids = r.lists.ids + (int64_t)row * r.top;
    float* weight = r.lists.weight + (int64_t)row * r.top;
    if (r.experts <= RANK_MAX) {
        for (int e = lane; e < r.experts; e += 32) {
            const float v = choice[e];
            int rank = 0;
#pragma unroll 8
            for (int i = 0; i < r.experts; i++) {
                const float o = choice[i];
                rank += o > v || (o == v && i < e);
            }
            if (rank < r.top) ids[rank] = e, weight[rank] = score(e);
        }
        return;
    }
    for (int k = 0; k < r.top; k++) {
        Best best{-INFINITY, 0x7fffffff};
        for (int e = lane; e < r.experts; e += 32) best = better(best, Best{choice[e], e});
        best = warp_best(best);
        const int e = min(best.i, r.experts - 1);
        if (lane == 0) {
            ids[k] = e, weight[k] = score(e);
            choice[e] = -INFINITY;
        }
        __syncwarp();
    }
}

__global__ void __launch_bounds__(ROUTE_WARPS * 32) route_kernel(const __grid_constant__ ExpertRouting r) {
    extern __shared__ float smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x * ROUTE_WARPS + warp;
    pdl_wait();
    pdl_launch_dependents();
    if (row < r.rows) route_row(r, row, smem + warp * (r.experts + r.groups), lane);
}

// Choice and lists of a small pass in one CTA, a warp per row.  The experts' counts, and ids of the pairs, in shared memory.
__global__ void __launch_bounds__(SMALL_ROWS * 32) route_small_kernel(const __grid_constant__ ExpertRouting r) {
    extern __shared__ float smem[];
    __shared__ int ids[SMALL_PAIRS], count[RANK_MAX], first[RANK_MAX + 1], chunk0[RANK_MAX + 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = r.rows * r.top;
    pdl_wait();
    pdl_launch_dependents();
    if (warp < r.rows) {
        route_row(r, warp, smem + warp * (r.experts + r.groups), lane);
        __syncwarp();
        for (int i = lane; i < r.top; i += 32) ids[warp * r.top + i] = r.lists.ids[warp * r.top + i];
    }
    if (threadIdx.x < r.experts) count[threadIdx.x] = 0;
    __syncthreads();
    if (threadIdx.x < n) atomicAdd(&count[ids[threadIdx.x]], 1);
    __syncthreads();
    if (threadIdx.x <= r.experts) {
        int s = 0, c = 0;
        for (int e = 0; e < (int)threadIdx.x; e++) s += count[e], c += (count[e] + r.chunk_slots - 1) / r.chunk_slots;
        first[threadIdx.x] = s, chunk0[threadIdx.x] = c;
        r.lists.first[threadIdx.x] = s;
        if (threadIdx.x == r.experts) *r.lists.n_chunks = c;
    }
    __syncthreads();
    if (threadIdx.x < n) {
        const int e = ids[threadIdx.x];
        int slot = first[e];
        for (int i = 0; i < (int)threadIdx.x; i++) slot += ids[i] == e;
        r.lists.slot_of[threadIdx.x] = slot, r.lists.token_of[slot] = threadIdx.x / r.top;
    }
    if (threadIdx.x < r.experts) {
        const int e = threadIdx.x, c0 = chunk0[e];
        for (int c = 0; c < chunk0[e + 1] - c0; c++)
            r.lists.chunks[c0 + c] = ExpertChunk{e, first[e] + c * r.chunk_slots, min(r.chunk_slots, count[e] - c * r.chunk_slots)};
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
    const int4* ids4 = reinterpret_cast<const int4*>(r.lists.ids);
    for (int i = threadIdx.x; i < n / 4; i += LIST_THREADS) {
        const int4 v = ids4[i];
        atomicAdd(&count[v.x], 1), atomicAdd(&count[v.y], 1), atomicAdd(&count[v.z], 1), atomicAdd(&count[v.w], 1);
    }
    for (int i = n / 4 * 4 + threadIdx.x; i < n; i += LIST_THREADS) atomicAdd(&count[r.lists.ids[i]], 1);
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
    // four neighbouring pairs per thread and step
    int at = slots;
    for (int i0 = 0; i0 < n; i0 += 4 * LIST_THREADS) {
        const int i = i0 + 4 * threadIdx.x;
        int id[4] = {-1, -1, -1, -1};
        if (i + 3 < n) {
            const int4 v = ids4[i / 4];
            id[0] = v.x, id[1] = v.y, id[2] = v.z, id[3] = v.w;
        } else {
            for (int k = 0; k < 4; k++)
                if (i + k < n) id[k] = r.lists.ids[i + k];
        }
        int mine_here = 0;
#pragma unroll
        for (int k = 0; k < 4; k++) mine_here += id[k] == e;
        int upto = mine_here;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int v = __shfl_up_sync(0xffffffffu, upto, o);
            if (lane >= o) upto += v;
        }
        __syncthreads();
        if (lane == 31) red[0][warp] = upto;
        __syncthreads();
        int before = upto - mine_here, all = 0;
#pragma unroll
        for (int w = 0; w < LIST_THREADS / 32; w++) {
            const int h = red[0][w];
            if (w < warp) before += h;
            all += h;
        }
#pragma unroll
        for (int k = 0; k < 4; k++)
            if (id[k] == e) {
                const int slot = at + before++;
                r.lists.slot_of[i + k] = slot, r.lists.token_of[slot] = (i + k) / r.top;
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
    if (r.rows <= SMALL_ROWS && r.rows * r.top <= SMALL_PAIRS && r.experts <= RANK_MAX) {
        const int threads = (std::max({r.rows * 32, r.experts + 1, r.rows * r.top}) + 31) / 32 * 32;
        return tsb_launch(ctx, route_small_kernel, dim3(1), dim3((unsigned)threads), (size_t)r.rows * (r.experts + r.groups) * sizeof(float), st, true, r);
    }
    cudaError_t e = tsb_launch(ctx, route_kernel, dim3((unsigned)((r.rows + ROUTE_WARPS - 1) / ROUTE_WARPS)), dim3(ROUTE_WARPS * 32),
                               (size_t)ROUTE_WARPS * (r.experts + r.groups) * sizeof(float), st, true, r);
    if (e != cudaSuccess) return e;
    return tsb_launch(ctx, expert_lists_kernel, dim3((unsigned)r.experts), dim3(LIST_THREADS), (size_t)r.experts * sizeof(int), st, true, r);
}

cudaError_t launch_gather_rows(tsb_ctx* ctx, cudaStream_t st, const void* x, int64_t x_bytes, const int32_t* token_of, int slots, void* out, int64_t bytes) {
    return tsb_launch(ctx, gather_rows_kernel, dim3((unsigned)slots), dim3(256), 0, st, true, (const uint8_t*)x, x_bytes, token_of, (uint8_t*)out, bytes);
}
