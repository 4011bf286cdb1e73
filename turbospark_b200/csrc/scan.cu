// Gated recurrences element by element (scan.cuh).
//
//   row by row   short portions: a thread per channel walks the portion's rows, eight of them in flight.
//   by chunks    long portions: a CTA owns CH channels of a chunk, 32 runs of a few rows.  A thread composes its run's rows into one step S -> A S + B; the
//                32 steps of a channel meet in shared memory, where a warp per channel scans them; then every thread walks its run from the state
//                before it.  Chunks with others behind them leave their step as a whole in a first launch, the second scans the steps before its own.
// f32 throughout.  A step is S + z (c - S), and a product of factors 1 - z is A - z A: where z is next to nothing the rounding of 1 - z would add up over a
// long memory.
#include <algorithm>

#include "recurrence_dev.cuh"
#include "scan.cuh"

namespace {

constexpr int ROWS_THREADS = 128, AHEAD = 8;
constexpr int RUNS = 32;  // of a chunk: the lanes of the warp that scans a channel

__device__ __forceinline__ void scan_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void scan_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
// 1 / (1 + e^-x): with bfloat16 outputs by the hardware's exponential and reciprocal (relative error a few 2^-22), in the f32 mode by the library's.
template <typename T>
__device__ __forceinline__ float sigmoid_of(float x) {
    if (sizeof(T) == 4) return rec_sigmoid(x);
    float e, y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * -1.4426950408889634f));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(1.f + e));
    return y;
}
template <typename T>
__device__ __forceinline__ float candidate(float u) {
    const float low = sigmoid_of<T>(u);
    return u >= 0.f ? u + 0.5f : low;
}

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
            s = fmaf(sigmoid_of<T>(x[i]), candidate<T>(u[i]) - s, s);
            scan_put(static_cast<T*>(g.out) + (int64_t)(p.row_first + t) * g.out_stride + c, s * o[i] * sigmoid_of<T>(o[i]));
            if (t + g.state.ring >= p.n_rows) state_at(g, rd.seq, pos0 + t)[c] = s;
        }
    }
}

// The gates of a thread's run, and the run as one step.
template <int RUN>
struct Run {
    float z[RUN], x[RUN];  // pre-activations, then z and c
    int n;                 // rows of the run that are there (may be negative)
    __device__ __forceinline__ void load(const GatedScan& g, int64_t row0, int c, int rows) {
        n = rows;
        const float* gate = g.gate + row0 * g.gate_stride + c;
#pragma unroll
        for (int i = 0; i < RUN; i++, gate += g.gate_stride) {
            z[i] = x[i] = 0.f;
            if (i < n) z[i] = gate[0], x[i] = gate[g.width];
        }
    }
    template <typename T>
    __device__ __forceinline__ float2 step() {
        float a = 1.f, b = 0.f;
#pragma unroll
        for (int i = 0; i < RUN; i++) {
            if (i >= n) continue;
            z[i] = sigmoid_of<T>(z[i]), x[i] = candidate<T>(x[i]);
            a = fmaf(-z[i], a, a), b = fmaf(z[i], x[i] - b, b);
        }
        return make_float2(a, b);
    }
};
// steps of the lanes composed with all that come before them
__device__ __forceinline__ float2 compose_before(float2 s, int lane) {
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
        const float pa = __shfl_up_sync(0xffffffffu, s.x, d), pb = __shfl_up_sync(0xffffffffu, s.y, d);
        if (lane >= d) s.y = fmaf(s.x, pb, s.y), s.x *= pa;
    }
    return s;
}
constexpr int RUN = SCAN_CHUNK / RUNS;

// What comes before a chunk, as steps: sums[chunk][channel] is the chunk before it as one step, and for a portion's first chunk the state before the portion (which
// the second launch, whose CTAs write states, could not read).
template <typename T, int CH>
__global__ void __launch_bounds__(CH * RUNS) scan_sums_kernel(const __grid_constant__ GatedScan g, const __grid_constant__ RowTiles chunks, float2* __restrict__ sums) {
    __shared__ float2 step[RUNS][CH + 1];
    const int ch = threadIdx.x % CH, run = threadIdx.x / CH, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x * CH + ch;
    const AttnTile p = row_tile(chunks, blockIdx.y);
    const int next = p.row_first + p.n_rows;
    const bool last = next >= g.n_rows || g.rows[next].slot == 0;
    const tsb_row_desc rd = g.rows[p.row_first];
    const bool ok = rd.seq >= 0 && rd.seq < g.state.n_streams;
    float2* out = sums + (int64_t)blockIdx.y * g.width;
    pdl_wait();
    pdl_launch_dependents();
    if (!ok) return;  // the second launch tells
    if (rd.slot == 0 && run == 0 && c < g.width) out[c] = make_float2(0.f, rd.base > 0 ? state_at(g, rd.seq, rd.base - 1)[c] : 0.f);
    if (last) return;
    Run<RUN> r;
    r.load(g, p.row_first + run * RUN, c, c < g.width ? RUN : 0);
    step[run][ch] = r.step<T>();
    __syncthreads();
    const float2 s = compose_before(step[lane][warp], lane);
    if (lane == 31 && blockIdx.x * CH + warp < g.width) out[g.width + blockIdx.x * CH + warp] = s;
}

template <typename T, int CH>
__global__ void __launch_bounds__(CH * RUNS) scan_chunks_kernel(const __grid_constant__ GatedScan g, const __grid_constant__ RowTiles chunks, const float2* __restrict__ sums,
                                                               uint32_t* __restrict__ err) {
    __shared__ float2 step[RUNS][CH + 1];
    __shared__ float before[RUNS][CH + 1];
    const int ch = threadIdx.x % CH, run = threadIdx.x / CH, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x * CH + ch, wc = blockIdx.x * CH + warp;  // the thread's channel, and the one its warp scans
    const AttnTile p = row_tile(chunks, blockIdx.y);
    const tsb_row_desc rd = g.rows[p.row_first];
    const int pos0 = rd.base + rd.slot, n_before = rd.slot / SCAN_CHUNK;  // chunks of the portion before this one
    const bool ok = rd.seq >= 0 && rd.seq < g.state.n_streams && n_before <= (int)blockIdx.y;
    if (!ok && threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
    const float carry = ok && !sums && wc < g.width && rd.base > 0 ? state_at(g, rd.seq, rd.base - 1)[wc] : 0.f;  // the portion is one chunk
    pdl_wait();
    pdl_launch_dependents();
    if (!ok) return;
    const int64_t row0 = p.row_first + run * RUN;
    Run<RUN> r;
    r.load(g, row0, c, c < g.width ? p.n_rows - run * RUN : 0);
    float o[RUN];
    const T* gate = static_cast<const T*>(g.out_gate) + row0 * g.out_gate_stride + c;
#pragma unroll
    for (int i = 0; i < RUN; i++, gate += g.out_gate_stride) o[i] = i < r.n ? rec_get(gate) : 0.f;
    // what comes before, 32 steps at a time
    float start = carry;
    for (int k0 = 0; sums && k0 <= n_before; k0 += 32) {
        float2 s = make_float2(1.f, 0.f);
        if (k0 + lane <= n_before && wc < g.width) s = __ldcg(sums + (int64_t)(blockIdx.y - n_before + k0 + lane) * g.width + wc);
        s = compose_before(s, lane);
        start = __shfl_sync(0xffffffffu, fmaf(s.x, start, s.y), 31);
    }
    step[run][ch] = r.step<T>();
    __syncthreads();
    {
        const float2 s = compose_before(step[lane][warp], lane);
        const float end = fmaf(s.x, start, s.y), prev = __shfl_up_sync(0xffffffffu, end, 1);
        before[lane][warp] = lane == 0 ? start : prev;
    }
    __syncthreads();
    float s = before[run][ch];
    T* out = static_cast<T*>(g.out) + row0 * g.out_stride + c;
#pragma unroll
    for (int i = 0; i < RUN; i++, out += g.out_stride) {
        if (i >= r.n) continue;
        s = fmaf(r.z[i], r.x[i] - s, s);
        r.x[i] = s;
        scan_put(out, s * o[i] * sigmoid_of<T>(o[i]));
    }
    auto kept = [&](int row) { return row + g.state.ring >= g.n_rows || g.rows[row + g.state.ring].seq != rd.seq; };  // one of the portion's last rows
    if (!kept(p.row_first + p.n_rows - 1)) return;
#pragma unroll
    for (int i = 0; i < RUN; i++)
        if (i < r.n && kept((int)row0 + i)) state_at(g, rd.seq, pos0 + run * RUN + i)[c] = r.x[i];
}

template <typename T, int CH>
cudaError_t launch_chunks(tsb_ctx* ctx, cudaStream_t st, const GatedScan& g, const RowTiles& chunks, bool several, float2* sums) {
    const dim3 grid((unsigned)((g.width + CH - 1) / CH), (unsigned)chunks.n);
    if (several)
        if (cudaError_t e = tsb_launch(ctx, scan_sums_kernel<T, CH>, grid, dim3(CH * RUNS), 0, st, true, g, chunks, sums); e != cudaSuccess) return e;
    return tsb_launch(ctx, scan_chunks_kernel<T, CH>, grid, dim3(CH * RUNS), 0, st, true, g, chunks, (const float2*)(several ? sums : nullptr), ctx->dev_error);
}

}  // namespace

cudaError_t launch_gated_scan_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const GatedScan& g, const RowTiles& portions) {
    if (portions.n == 0) return cudaSuccess;
    auto run = [&](auto kernel) {
        return tsb_launch(ctx, kernel, dim3((unsigned)((g.width + ROWS_THREADS - 1) / ROWS_THREADS), (unsigned)portions.n), dim3(ROWS_THREADS), 0, st, true, g, portions, ctx->dev_error);
    };
    return f32 ? run(scan_rows_kernel<float>) : run(scan_rows_kernel<__nv_bfloat16>);
}

cudaError_t launch_gated_scan_chunks(tsb_ctx* ctx, cudaStream_t st, bool f32, const GatedScan& g, const RowTiles& chunks, bool several, float2* sums) {
    if (chunks.n == 0) return cudaSuccess;
    return f32 ? launch_chunks<float, 16>(ctx, st, g, chunks, several, sums) : launch_chunks<__nv_bfloat16, 16>(ctx, st, g, chunks, several, sums);
}
