// Gated recurrences element by element (scan.cuh).
//
//   scan_rows_kernel  short portions: a thread per channel walks the portion's rows, eight of them in flight.
//   scan_kernel       long portions: a CTA owns CH channels of a portion and goes through it in batches of 32 runs of RUN rows.  A thread composes
//                     its run's rows into one step S -> A S + B; the 32 steps of a channel meet in shared memory, where a warp per channel scans
//                     them; then every thread walks its run from the state before it.  Gates are read once and stay in registers.
// f32 throughout.  1 - z is sigmoid(-x), not a difference, and a step is S + z (c - S): close to zero or one the rounding of z would
// otherwise add up over a long memory.
#include <algorithm>

#include "recurrence_dev.cuh"
#include "scan.cuh"

namespace {

constexpr int ROWS_THREADS = 128, AHEAD = 8;
constexpr int RUNS = 32;  // of a batch: the lanes of the warp that scans a channel

__device__ __forceinline__ void scan_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void scan_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float candidate(float u) { return u >= 0.f ? u + 0.5f : rec_sigmoid(u); }

__device__ __forceinline__ float* state_at(const GatedScan& g, int seq, int pos) {
    return g.state.s + ((int64_t)seq * g.state.ring + (pos & (g.state.ring - 1))) * recurrence_v_pitch(g.width);
}

template <typename T>
__global__ void __launch_bounds__(ROWS_THREADS) scan_rows_kernel(const __grid_constant__ GatedScan g, const __grid_constant__ RowTiles portions, uint32_t* __restrict__ err) {
    const int c = blockIdx.x * ROWS_THREADS + threadIdx.x;
    const AttnTile p = row_tile(portions, blockIdx.y);
    const tsb_row_desc rd = g.rows[p.row_first];
    const int pos0 = rd.base + rd.slot;
    const bool ok = rd.seq >= 0 && rd.seq < g.state.n_streams;
    if (!ok && threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
    float s = ok && c < g.width && pos0 > 0 ? state_at(g, rd.seq, pos0 - 1)[c] : 0.f;  // of an earlier pass
    pdl_wait();
    pdl_launch_dependents();
    if (!ok || c >= g.width) return;
    for (int t0 = 0; t0 < p.n_rows; t0 += AHEAD) {
        float x[AHEAD], u[AHEAD], o[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; i++)
            if (t0 + i < p.n_rows) {
                const int64_t row = p.row_first + t0 + i;
                x[i] = g.gate[row * g.gate_stride + c], u[i] = g.gate[row * g.gate_stride + g.width + c];
                o[i] = rec_get(static_cast<const T*>(g.out_gate) + row * g.out_gate_stride + c);
            }
#pragma unroll
        for (int i = 0; i < AHEAD; i++) {
            const int t = t0 + i;
            if (t >= p.n_rows) break;
            s = fmaf(rec_sigmoid(x[i]), candidate(u[i]) - s, s);
            scan_put(static_cast<T*>(g.out) + (int64_t)(p.row_first + t) * g.out_stride + c, s * rec_silu(o[i]));
            if (t + g.state.ring >= p.n_rows) state_at(g, rd.seq, pos0 + t)[c] = s;
        }
    }
}

template <typename T, int CH, int RUN>
__global__ void __launch_bounds__(CH * RUNS) scan_kernel(const __grid_constant__ GatedScan g, const __grid_constant__ RowTiles portions, uint32_t* __restrict__ err) {
    __shared__ float2 step[RUNS][CH + 1];
    __shared__ float before[RUNS][CH + 1], carry[CH];
    const int ch = threadIdx.x % CH, run = threadIdx.x / CH, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x * CH + ch;
    const AttnTile p = row_tile(portions, blockIdx.y);
    const tsb_row_desc rd = g.rows[p.row_first];
    const int pos0 = rd.base + rd.slot;
    const bool ok = rd.seq >= 0 && rd.seq < g.state.n_streams, in = ok && c < g.width;
    if (!ok && threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
    if (run == 0) carry[ch] = in && pos0 > 0 ? state_at(g, rd.seq, pos0 - 1)[c] : 0.f;
    pdl_wait();
    pdl_launch_dependents();
    if (!ok) return;
    for (int b0 = 0; b0 < p.n_rows; b0 += RUNS * RUN) {
        const int t0 = b0 + run * RUN, n = in ? min(RUN, p.n_rows - t0) : 0;  // may be negative
        const int64_t row0 = p.row_first + t0;
        float z[RUN], x[RUN], o[RUN];
#pragma unroll
        for (int i = 0; i < RUN; i++) {
            z[i] = x[i] = o[i] = 0.f;
            if (i < n) {
                const float* gate = g.gate + (row0 + i) * g.gate_stride + c;
                z[i] = gate[0], x[i] = gate[g.width];
                o[i] = rec_get(static_cast<const T*>(g.out_gate) + (row0 + i) * g.out_gate_stride + c);
            }
        }
        float a = 1.f, b = 0.f;
#pragma unroll
        for (int i = 0; i < RUN; i++) {
            if (i >= n) continue;
            const float left = rec_sigmoid(-z[i]);
            z[i] = rec_sigmoid(z[i]), x[i] = candidate(x[i]);
            a *= left, b = fmaf(z[i], x[i] - b, b);
        }
        step[run][ch] = make_float2(a, b);
        __syncthreads();
        {
            // warp = channel, lane = run: steps composed with all that come before
            float2 s = step[lane][warp];
#pragma unroll
            for (int d = 1; d < 32; d <<= 1) {
                const float pa = __shfl_up_sync(0xffffffffu, s.x, d), pb = __shfl_up_sync(0xffffffffu, s.y, d);
                if (lane >= d) s.y = fmaf(s.x, pb, s.y), s.x *= pa;
            }
            const float start = carry[warp], end = fmaf(s.x, start, s.y), prev = __shfl_up_sync(0xffffffffu, end, 1);
            before[lane][warp] = lane == 0 ? start : prev;
            __syncwarp();
            if (lane == 31) carry[warp] = end;
        }
        __syncthreads();
        float s = before[run][ch];
#pragma unroll
        for (int i = 0; i < RUN; i++) {
            if (i >= n) continue;
            s = fmaf(z[i], x[i] - s, s);
            scan_put(static_cast<T*>(g.out) + (row0 + i) * g.out_stride + c, s * rec_silu(o[i]));
            if (t0 + i + g.state.ring >= p.n_rows) state_at(g, rd.seq, pos0 + t0 + i)[c] = s;
        }
    }
}

template <typename T>
cudaError_t launch_of(tsb_ctx* ctx, cudaStream_t st, const GatedScan& g, const RowTiles& portions) {
    if (portions.longest < SCAN_MIN_ROWS)
        return tsb_launch(ctx, scan_rows_kernel<T>, dim3((unsigned)((g.width + ROWS_THREADS - 1) / ROWS_THREADS), (unsigned)portions.n), dim3(ROWS_THREADS), 0, st, true, g, portions,
                          ctx->dev_error);
    auto run = [&](auto kernel, int ch) {
        return tsb_launch(ctx, kernel, dim3((unsigned)((g.width + ch - 1) / ch), (unsigned)portions.n), dim3(ch * RUNS), 0, st, true, g, portions, ctx->dev_error);
    };
    // fewer channels per CTA where whole sectors of them would leave SMs idle
    const int64_t ctas = (int64_t)portions.n * ((g.width + 15) / 16);
    return ctas < ctx->sm_count ? run(scan_kernel<T, 8, 4>, 8) : run(scan_kernel<T, 16, 4>, 16);
}

}  // namespace

cudaError_t launch_gated_scan(tsb_ctx* ctx, cudaStream_t st, bool f32, const GatedScan& g, const RowTiles& portions) {
    if (portions.n == 0) return cudaSuccess;
    return f32 ? launch_of<float>(ctx, st, g, portions) : launch_of<__nv_bfloat16>(ctx, st, g, portions);
}
