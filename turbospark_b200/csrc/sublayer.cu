// Row operators around the sublayers of output-norm layers (sublayer.cuh).
#include <cuda_bf16.h>

#include <algorithm>
#include <type_traits>

#include "sublayer.cuh"

namespace {

constexpr int THREADS = 256, WARPS = THREADS / 32;

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// W (1 or 4) neighbouring numbers
template <int W>
struct Vec {
    float v[W];
};
template <int W>
__device__ __forceinline__ Vec<W> zeros() {
    Vec<W> r;
#pragma unroll
    for (int i = 0; i < W; i++) r.v[i] = 0.f;
    return r;
}
__device__ __forceinline__ Vec<1> load(const float* p, Vec<1>) { return Vec<1>{{*p}}; }
__device__ __forceinline__ Vec<4> load(const float* p, Vec<4>) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    return Vec<4>{{f.x, f.y, f.z, f.w}};
}
__device__ __forceinline__ Vec<1> load(const __nv_bfloat16* p, Vec<1>) { return Vec<1>{{__bfloat162float(*p)}}; }
__device__ __forceinline__ Vec<4> load(const __nv_bfloat16* p, Vec<4>) {
    const uint2 w = *reinterpret_cast<const uint2*>(p);
    return Vec<4>{{__uint_as_float(w.x << 16), __uint_as_float(w.x & 0xFFFF0000u), __uint_as_float(w.y << 16), __uint_as_float(w.y & 0xFFFF0000u)}};
}
__device__ __forceinline__ void store(float* p, const Vec<1>& a) { *p = a.v[0]; }
__device__ __forceinline__ void store(float* p, const Vec<4>& a) { *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]); }
__device__ __forceinline__ void store(__nv_bfloat16* p, const Vec<1>& a) { *p = __float2bfloat16_rn(a.v[0]); }
__device__ __forceinline__ void store(__nv_bfloat16* p, const Vec<4>& a) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a.v[0], a.v[1]), hi = __floats2bfloat162_rn(a.v[2], a.v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
// bfloat16 results take the fast exponential and division (relative error a few 2^-22)
template <typename T>
__device__ __forceinline__ float silu(float z) {
    return sizeof(T) == 4 ? z * sigmoid(z) : __fdividef(z, 1.f + __expf(-z));
}

// 1 / rms of the group that column c belongs to, from the columns' squares.  One of NT threads holds columns (k * NT + thread) * W + i, k < V.
// FAST: groups are multiples of 32 W columns, so a warp's columns of one k share a group and the whole reduction takes one barrier.
// sq: shared memory, two of them used in turn (call with parity 0, 1, 0, ...).
template <int NT, int V, int W, bool FAST>
struct GroupNorm {
    static constexpr int NW = NT / 32;
    int d, width, groups;
    float eps;
    float *sq, *sums;  // FAST: [2][V * NW]; else sq [d / W], sums [groups]
    __device__ __forceinline__ void rms(const Vec<W> (&x)[V], int parity, float (&inv)[V]) const {
        float s[V];
#pragma unroll
        for (int k = 0; k < V; k++) {
            s[k] = 0.f;
#pragma unroll
            for (int i = 0; i < W; i++) s[k] = fmaf(x[k].v[i], x[k].v[i], s[k]);
        }
        const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
        if (FAST) {
            float* red = sq + parity * V * NW;
#pragma unroll
            for (int k = 0; k < V; k++) {
                const float t = warp_sum(s[k]);
                if (lane == 0) red[k * NW + warp] = t;
            }
            __syncthreads();
            const int per = width / (32 * W);  // warp runs per group
#pragma unroll
            for (int k = 0; k < V; k++) {
                const int g = (k * NW + warp) / per;
                float t = 0.f;
                if ((k * NT + (int)threadIdx.x) * W < d)
                    for (int i = 0; i < per; i++) t += red[g * per + i];
                inv[k] = 1.f / sqrtf(t / (float)width + eps);
            }
        } else {
#pragma unroll
            for (int k = 0; k < V; k++) {
                const int u = k * NT + threadIdx.x;
                if (u * W < d) sq[u] = s[k];
            }
            __syncthreads();
            const int per = width / W;
            for (int g = warp; g < groups; g += NW) {
                float t = 0.f;
                for (int i = lane; i < per; i += 32) t += sq[g * per + i];
                t = warp_sum(t);
                if (lane == 0) sums[g] = 1.f / sqrtf(t / (float)width + eps);
            }
            __syncthreads();
#pragma unroll
            for (int k = 0; k < V; k++) {
                const int c = (k * NT + threadIdx.x) * W;
                inv[k] = c < d ? sums[c / width] : 0.f;
            }
            // the next call's first barrier separates its writes of sums from these reads; sq is rewritten only behind the second one above
        }
    }
};
template <int NT, int V, int W>
size_t group_norm_smem(int d, int groups, bool fast) {
    return (fast ? (size_t)2 * V * (NT / 32) : (size_t)(d / W + groups)) * sizeof(float);
}

// ------------------------------------------------------------------ end of a sublayer
enum SublayerSource { FROM_Y, FROM_EXPERTS, FROM_TABLE };

template <typename T, int NT, int V, int W, bool FAST, int TM>
__global__ void __launch_bounds__(NT) sublayer_end_kernel(const __grid_constant__ SublayerEnd s, uint32_t* __restrict__ err) {
    extern __shared__ float smem[];
    const AttnTile tile = row_tile(s.tiles, blockIdx.x);
    const tsb_row_desc rd = s.rows[tile.row_first];
    const int d = s.d, halo = s.taps > 0 ? min(s.taps - 1, rd.slot) : 0;
    const bool ok = s.taps <= 1 || (rd.seq >= 0 && rd.seq < s.ring.n_streams);
    GroupNorm<NT, V, W, FAST> norm;
    norm.d = d, norm.groups = s.groups, norm.width = d / s.groups, norm.eps = s.eps, norm.sq = smem, norm.sums = smem + d / W;
    Vec<W> hist[TM > 1 ? TM - 1 : 1][V];  // hist[j]: the row j + 1 before the current one
    Vec<W> w[V];
#pragma unroll
    for (int k = 0; k < V; k++) {
        const int c = (k * NT + threadIdx.x) * W;
        w[k] = c < d && s.norm_w ? load(s.norm_w + c, Vec<W>()) : zeros<W>();
    }
    Vec<W> taps[TM][V];  // taps[j]: of the row j before
#pragma unroll
    for (int j = 0; j < TM; j++)
#pragma unroll
        for (int k = 0; k < V; k++) {
            const int c = (k * NT + threadIdx.x) * W;
            taps[j][k] = j < s.taps && c < d ? load(s.taps_w + (int64_t)(s.taps - 1 - j) * d + c, Vec<W>()) : zeros<W>();
        }
    pdl_wait();
    pdl_launch_dependents();
    if (!ok) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        return;
    }
    const int first = tile.row_first - halo, pos_first = rd.base + rd.slot - halo;
#pragma unroll
    for (int j = 0; j < TM - 1; j++) {
        const int pos = pos_first - 1 - j;
        const bool in = j < s.taps - 1 - halo && pos >= 0;  // fewer halo rows than taps: the portion starts at `first`
        const float* p = in ? ring_row_before(s.ring, rd.seq, rd.base, pos, s.use_before) : nullptr;
#pragma unroll
        for (int k = 0; k < V; k++) {
            const int c = (k * NT + threadIdx.x) * W;
            hist[j][k] = in && c < d ? load(p + c, Vec<W>()) : zeros<W>();
        }
    }
    // the sublayer's output and the stream of a row; those of the next row are under way while a row is normed
    Vec<W> y_next[V], x_next[V];
    auto fetch = [&](int r) {
#pragma unroll
        for (int k = 0; k < V; k++) {
            const int c = (k * NT + threadIdx.x) * W;
            x_next[k] = c < d ? load(s.x_in + (int64_t)r * d + c, Vec<W>()) : zeros<W>();
            y_next[k] = s.y && c < d ? load(s.y + (int64_t)r * d + c, Vec<W>()) : zeros<W>();
        }
        if (s.y) return;
        constexpr int AT_ONCE = V * W <= 8 ? 4 : 2;  // expert rows in flight
        for (int e0 = 0; e0 < s.top; e0 += AT_ONCE) {
            float f[AT_ONCE];
            Vec<W> v[AT_ONCE][V];
#pragma unroll
            for (int e = 0; e < AT_ONCE; e++) {
                const int64_t at = (int64_t)r * s.top + e0 + e;
                const bool in = e0 + e < s.top;
                f[e] = in ? s.weight[at] : 0.f;
                const T* row = static_cast<const T*>(s.experts) + (int64_t)(in ? s.slot_of[at] : 0) * s.expert_stride;
#pragma unroll
                for (int k = 0; k < V; k++) {
                    const int c = (k * NT + threadIdx.x) * W;
                    v[e][k] = in && c < d ? load(row + c, Vec<W>()) : zeros<W>();
                }
            }
#pragma unroll
            for (int e = 0; e < AT_ONCE; e++)
#pragma unroll
                for (int k = 0; k < V; k++)
#pragma unroll
                    for (int i = 0; i < W; i++) y_next[k].v[i] = fmaf(f[e], v[e][k].v[i], y_next[k].v[i]);
        }
    };
    const int last = tile.row_first + tile.n_rows - 1;
    const bool any_kept = s.taps > 1 && ring_keeps(s.ring, s.rows, s.n_rows, last, rd.seq);
    if (!s.table) fetch(first);
    for (int r = first, parity = 0; r <= last; r++, parity ^= 1) {
        Vec<W> x[V];
        if (s.table) {
            const int tok = s.tokens[(int64_t)r * s.token_stride], pos = pos_first + (r - first);
            const bool bad = tok < 0 || tok >= s.vocab || (s.positions && pos >= s.n_positions);
            if (bad && threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
#pragma unroll
            for (int k = 0; k < V; k++) {
                const int c = (k * NT + threadIdx.x) * W;
                x[k] = zeros<W>();
                if (bad || c >= d) continue;
                x[k] = load(static_cast<const T*>(s.table) + (int64_t)tok * d + c, Vec<W>());
                const Vec<W> p = s.positions ? load(static_cast<const T*>(s.positions) + (int64_t)pos * d + c, Vec<W>()) : zeros<W>();
#pragma unroll
                for (int i = 0; i < W; i++) x[k].v[i] = fmaf(s.embed_scale, x[k].v[i], p.v[i]);
            }
        } else {
            Vec<W> y[V];
#pragma unroll
            for (int k = 0; k < V; k++) x[k] = x_next[k], y[k] = y_next[k];
            if (r < last) fetch(r + 1);
            float inv[V];
            norm.rms(y, parity, inv);
#pragma unroll
            for (int k = 0; k < V; k++)
#pragma unroll
                for (int i = 0; i < W; i++) x[k].v[i] = fmaf(y[k].v[i] * inv[k], w[k].v[i], x[k].v[i]);
        }
        if (r >= tile.row_first) {
            float* keep = nullptr;
            if (any_kept && ring_keeps(s.ring, s.rows, s.n_rows, r, rd.seq)) keep = ring_row(s.ring, rd.seq, pos_first + (r - first));
#pragma unroll
            for (int k = 0; k < V; k++) {
                const int c = (k * NT + threadIdx.x) * W;
                if (c >= d) continue;
                store(s.x_out + (int64_t)r * d + c, x[k]);
                if (s.taps == 0) continue;
                if (keep) store(keep + c, x[k]);
                Vec<W> o;
#pragma unroll
                for (int i = 0; i < W; i++) {
                    o.v[i] = fmaf(taps[0][k].v[i], x[k].v[i], x[k].v[i]);
#pragma unroll
                    for (int j = 0; j < TM - 1; j++) o.v[i] = fmaf(taps[j + 1][k].v[i], hist[j][k].v[i], o.v[i]);
                }
                store(static_cast<T*>(s.out) + (int64_t)r * s.out_stride + c, o);
            }
        }
#pragma unroll
        for (int j = TM - 2; j > 0; j--)
#pragma unroll
            for (int k = 0; k < V; k++) hist[j][k] = hist[j - 1][k];
        if (TM > 1) {
#pragma unroll
            for (int k = 0; k < V; k++) hist[0][k] = x[k];
        }
    }
}

__global__ void __launch_bounds__(THREADS)
    rings_before_kernel(const RowRing* __restrict__ rings, const tsb_row_desc* __restrict__ rows, const __grid_constant__ RowTiles portions) {
    pdl_wait();
    pdl_launch_dependents();
    const tsb_row_desc rd = rows[row_tile(portions, blockIdx.x).row_first];
    const RowRing r = rings[blockIdx.y];
    if (rd.slot != 0 || rd.seq < 0 || rd.seq >= r.n_streams) return;
    for (int k = 0; k < r.keep; k++) {
        const int pos = rd.base - r.keep + k;
        if (pos < 0) continue;
        const float* src = ring_row(r, rd.seq, pos);
        float* dst = r.before + ((int64_t)rd.seq * r.keep + k) * r.width;
        for (int i = threadIdx.x; i < r.width; i += THREADS) dst[i] = src[i];
    }
}

template <typename T, int V, int W, bool FAST>
__global__ void __launch_bounds__(THREADS)
    group_norm_rows_kernel(const float* x, int d, const float* __restrict__ weight, int groups, float eps, const int32_t* __restrict__ want, int want_first,
                           int want_step, T* out, int64_t out_stride) {
    extern __shared__ float smem[];
    pdl_wait();
    pdl_launch_dependents();
    const int r = want ? want[blockIdx.x] : (int)blockIdx.x * want_step + want_first;
    GroupNorm<THREADS, V, W, FAST> norm;
    norm.d = d, norm.groups = groups, norm.width = d / groups, norm.eps = eps, norm.sq = smem, norm.sums = smem + d / W;
    Vec<W> v[V];
    float inv[V];
#pragma unroll
    for (int k = 0; k < V; k++) {
        const int c = (k * THREADS + threadIdx.x) * W;
        v[k] = c < d ? load(x + (int64_t)r * d + c, Vec<W>()) : zeros<W>();
    }
    norm.rms(v, 0, inv);
#pragma unroll
    for (int k = 0; k < V; k++) {
        const int c = (k * THREADS + threadIdx.x) * W;
        if (c >= d) continue;
        const Vec<W> w = load(weight + c, Vec<W>());
#pragma unroll
        for (int i = 0; i < W; i++) v[k].v[i] *= inv[k] * w.v[i];
        store(out + (int64_t)blockIdx.x * out_stride + c, v[k]);
    }
}

// ------------------------------------------------------------------ norms of whole projections
// blockIdx.y: queries or keys of the row.
template <typename T, int W>
__global__ void __launch_bounds__(THREADS) projection_norms_kernel(const __grid_constant__ ProjectionNorms p, uint32_t* __restrict__ err) {
    __shared__ float red[WARPS];
    const bool query = blockIdx.y == 0;
    const int r = blockIdx.x, heads = query ? p.n_q : p.n_k, n = heads * p.width;
    const tsb_row_desc rd = p.rows[r];
    const float *src = p.raw + (int64_t)r * p.raw_stride + (query ? 0 : (int64_t)p.n_q * p.width), *w = query ? p.q_weight : p.k_weight;
    pdl_wait();
    pdl_launch_dependents();
    constexpr int HELD = 4;  // vectors that stay in registers
    Vec<W> held[HELD];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < HELD; k++) {
        const int i = (k * THREADS + threadIdx.x) * W;
        held[k] = i < n ? load(src + i, Vec<W>()) : zeros<W>();
    }
#pragma unroll
    for (int k = 0; k < HELD; k++)
#pragma unroll
        for (int j = 0; j < W; j++) ss = fmaf(held[k].v[j], held[k].v[j], ss);
    for (int i = (HELD * THREADS + threadIdx.x) * W; i < n; i += THREADS * W) {
        const Vec<W> v = load(src + i, Vec<W>());
#pragma unroll
        for (int j = 0; j < W; j++) ss = fmaf(v.v[j], v.v[j], ss);
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < WARPS; i++) ss += red[i];
    const float f = 1.f / sqrtf(ss / (float)n + p.eps);
    T* dst;
    int step = p.width;
    if (query) {
        dst = static_cast<T*>(p.q) + (int64_t)r * p.q_stride, step = p.q_step;
    } else {
        dst = key_row<T>(p.keys, rd.seq, rd.base + rd.slot);
        if (!dst) {
            if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
            return;
        }
        step = p.keys.head_step;
    }
    auto finish = [&](int i, Vec<W> v) {
        const Vec<W> g = load(w + i, Vec<W>());
#pragma unroll
        for (int j = 0; j < W; j++) v.v[j] *= f * g.v[j];
        const int at = i % p.width;
        if (p.rot) {
#pragma unroll
            for (int j = 0; j < W; j++) {
                const int c = at + j;
                if (c >= 2 * p.rot_half || (W > 1 && (j & 1))) continue;
                const float2 t = p.rot[(int64_t)r * p.rot_half + (c >> 1)];
                if (W == 1) {  // the other column of the pair is another thread's
                    const int other = i - at + (at ^ 1);
                    const float o = src[other] * f * w[other];
                    v.v[0] = c & 1 ? fmaf(v.v[0], t.x, o * t.y) : fmaf(v.v[0], t.x, -o * t.y);
                } else {
                    const float a = v.v[j], b = v.v[(j + 1) % W];
                    v.v[j] = fmaf(a, t.x, -b * t.y), v.v[(j + 1) % W] = fmaf(b, t.x, a * t.y);
                }
            }
        }
        store(dst + (int64_t)(i / p.width) * step + at, v);
    };
#pragma unroll
    for (int k = 0; k < HELD; k++)
        if ((k * THREADS + (int)threadIdx.x) * W < n) finish((k * THREADS + threadIdx.x) * W, held[k]);
    for (int i = (HELD * THREADS + threadIdx.x) * W; i < n; i += THREADS * W) finish(i, load(src + i, Vec<W>()));
    if (query && step > p.width) {
        const int tail = step - p.width;
        for (int i = threadIdx.x; i < heads * tail; i += THREADS) put(dst + (int64_t)(i / tail) * step + p.width + i % tail, 0.f);
    }
}

// ------------------------------------------------------------------ short convolution
// A thread owns W channels and walks the rows of its tile with the rows before in registers.
// RESIDUAL: `in` (f32) itself is added, and there is neither bias nor activation.
template <typename T, int W, int TM, bool RESIDUAL>
__global__ void __launch_bounds__(THREADS) short_conv_kernel(const __grid_constant__ ShortConv s, uint32_t* __restrict__ err) {
    const AttnTile tile = row_tile(s.tiles, blockIdx.x);
    const tsb_row_desc rd = s.rows[tile.row_first];
    const int c = (blockIdx.y * THREADS + threadIdx.x) * W;
    const bool ok = rd.seq >= 0 && rd.seq < s.ring.n_streams;
    pdl_wait();
    pdl_launch_dependents();
    if (!ok && threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
    if (!ok || c >= s.channels) return;
    Vec<W> w[TM], hist[TM - 1];
    const Vec<W> bias = RESIDUAL ? zeros<W>() : load(s.bias + c, Vec<W>());
#pragma unroll
    for (int j = 0; j < TM; j++) w[j] = j < s.taps ? load(s.w + (int64_t)(s.taps - 1 - j) * s.channels + c, Vec<W>()) : zeros<W>();  // w[j]: j rows back
    using In = std::conditional_t<RESIDUAL, float, T>;
    const In* in = static_cast<const In*>(s.in) + c;
#pragma unroll
    for (int j = 0; j < TM - 1; j++) {
        const int back = j + 1, pos = rd.base + rd.slot - back;
        hist[j] = zeros<W>();
        if (back >= s.taps || pos < 0) continue;
        hist[j] = back <= rd.slot ? load(in + (int64_t)(tile.row_first - back) * s.in_stride, Vec<W>())
                                  : load(ring_row_before(s.ring, rd.seq, rd.base, pos, s.use_before) + c, Vec<W>());
    }
    constexpr int AHEAD = W == 4 ? 4 : 8;  // rows in flight
    for (int i0 = 0; i0 < tile.n_rows; i0 += AHEAD) {
        Vec<W> x[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; i++)
            if (i0 + i < tile.n_rows) x[i] = load(in + (int64_t)(tile.row_first + i0 + i) * s.in_stride, Vec<W>());
        const bool any_kept = s.taps > 1 && ring_keeps(s.ring, s.rows, s.n_rows, tile.row_first + tile.n_rows - 1, rd.seq);
#pragma unroll
        for (int i = 0; i < AHEAD; i++) {
            if (i0 + i >= tile.n_rows) break;
            const int r = tile.row_first + i0 + i;
            if (any_kept && ring_keeps(s.ring, s.rows, s.n_rows, r, rd.seq)) store(ring_row(s.ring, rd.seq, rd.base + rd.slot + i0 + i) + c, x[i]);
            Vec<W> o = RESIDUAL ? x[i] : bias;
#pragma unroll
            for (int k = 0; k < W; k++) {
#pragma unroll
                for (int j = TM - 2; j >= 0; j--) o.v[k] = fmaf(w[j + 1].v[k], hist[j].v[k], o.v[k]);
                o.v[k] = fmaf(w[0].v[k], x[i].v[k], o.v[k]);
                if (!RESIDUAL) o.v[k] = silu<T>(o.v[k]);
            }
            store(static_cast<T*>(s.out) + (int64_t)r * s.out_stride + c, o);
#pragma unroll
            for (int j = TM - 2; j > 0; j--) hist[j] = hist[j - 1];
            hist[0] = x[i];
        }
    }
}

// ------------------------------------------------------------------ gated norm of a recurrence's output
template <typename T, int W>
__global__ void __launch_bounds__(THREADS) gated_norm_kernel(const __grid_constant__ GatedNorm g) {
    extern __shared__ float smem[];
    float *v = smem, *sq = smem + g.width, *inv = sq + g.width / W;
    const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gw = g.width / g.groups;
    pdl_wait();
    pdl_launch_dependents();
    for (int c = threadIdx.x * W; c < g.width; c += THREADS * W) {
        Vec<W> x = load(g.o + (int64_t)r * g.o_stride + c, Vec<W>());
        if (g.pre_gate) {
            const Vec<W> z = load(static_cast<const T*>(g.pre_gate) + (int64_t)r * g.gate_stride + c, Vec<W>());
#pragma unroll
            for (int i = 0; i < W; i++) x.v[i] *= silu<T>(z.v[i]);
        }
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < W; i++) s = fmaf(x.v[i], x.v[i], s);
        store(v + c, x);
        sq[c / W] = s;
    }
    __syncthreads();
    const int per = gw / W;
    for (int k = warp; k < g.groups; k += WARPS) {
        float s = 0.f;
        for (int i = lane; i < per; i += 32) s += sq[k * per + i];
        s = warp_sum(s);
        if (lane == 0) inv[k] = g.scale / sqrtf(s / (float)gw + g.eps);
    }
    __syncthreads();
    for (int c = threadIdx.x * W; c < g.width; c += THREADS * W) {
        Vec<W> x = load(v + c, Vec<W>());
        const Vec<W> w = load(g.weight + c % g.weight_n, Vec<W>());
        const float f = inv[c / gw];
#pragma unroll
        for (int i = 0; i < W; i++) x.v[i] *= f * w.v[i];
        if (g.post_gate) {
            const Vec<W> z = load(static_cast<const T*>(g.post_gate) + (int64_t)r * g.gate_stride + c, Vec<W>());
#pragma unroll
            for (int i = 0; i < W; i++) x.v[i] *= sigmoid(z.v[i]);
        }
        store(static_cast<T*>(g.out) + (int64_t)r * g.out_stride + c, x);
    }
}

// columns per thread and how many of them at a time: (4, V) when groups and strides are whole vectors
constexpr int MAX_VECS4 = 8, MAX_VECS1 = 16;
bool by_fours(int d, int groups) { return (d / groups) % 4 == 0 && d <= 4 * THREADS * MAX_VECS4; }

template <typename T, int NT, int V, int W, bool FAST>
cudaError_t launch_end(tsb_ctx* ctx, cudaStream_t st, const SublayerEnd& s) {
    const size_t smem = group_norm_smem<NT, V, W>(s.d, s.groups, FAST);
    auto run = [&](auto kernel) { return tsb_launch(ctx, kernel, dim3((unsigned)s.tiles.n), dim3(NT), smem, st, true, s, ctx->dev_error); };
    if (s.taps == 0) return run(sublayer_end_kernel<T, NT, V, W, FAST, 1>);
    return s.taps <= 4 ? run(sublayer_end_kernel<T, NT, V, W, FAST, 4>) : run(sublayer_end_kernel<T, NT, V, W, FAST, CONV_MAX_TAPS>);
}
template <typename T>
cudaError_t launch_end_of(tsb_ctx* ctx, cudaStream_t st, const SublayerEnd& s) {
    const int d = s.d, gw = d / s.groups;
    if (by_fours(d, s.groups) && s.out_stride % 4 == 0 && s.expert_stride % 4 == 0) {
        const bool fast = gw % 128 == 0;
        if (d <= 1024) return fast ? launch_end<T, 256, 1, 4, true>(ctx, st, s) : launch_end<T, 256, 1, 4, false>(ctx, st, s);
        if (d <= 2048) return fast ? launch_end<T, 512, 1, 4, true>(ctx, st, s) : launch_end<T, 512, 1, 4, false>(ctx, st, s);
        if (d <= 4096) return fast ? launch_end<T, 512, 2, 4, true>(ctx, st, s) : launch_end<T, 512, 2, 4, false>(ctx, st, s);
        return fast ? launch_end<T, 512, 4, 4, true>(ctx, st, s) : launch_end<T, 512, 4, 4, false>(ctx, st, s);
    }
    return d <= 1024 ? launch_end<T, 256, 4, 1, false>(ctx, st, s) : launch_end<T, 512, 8, 1, false>(ctx, st, s);
}

template <typename T>
cudaError_t launch_norm_of(tsb_ctx* ctx, cudaStream_t st, const float* x, int d, const float* weight, int groups, float eps, const int32_t* want, int first, int step, int n,
                           T* out, int64_t out_stride) {
    auto run = [&](auto kernel, size_t smem) {
        return tsb_launch(ctx, kernel, dim3((unsigned)n), dim3(THREADS), smem, st, true, x, d, weight, groups, eps, want, first, step, out, out_stride);
    };
    if (by_fours(d, groups) && out_stride % 4 == 0) {
        if ((d / groups) % 128 == 0) return run(group_norm_rows_kernel<T, MAX_VECS4, 4, true>, group_norm_smem<THREADS, MAX_VECS4, 4>(d, groups, true));
        return run(group_norm_rows_kernel<T, MAX_VECS4, 4, false>, group_norm_smem<THREADS, MAX_VECS4, 4>(d, groups, false));
    }
    return run(group_norm_rows_kernel<T, MAX_VECS1, 1, false>, group_norm_smem<THREADS, MAX_VECS1, 1>(d, groups, false));
}

template <bool RESIDUAL>
cudaError_t launch_conv(tsb_ctx* ctx, cudaStream_t st, bool f32, const ShortConv& c) {
    const bool vec = c.channels % 4 == 0 && c.in_stride % 4 == 0 && c.out_stride % 4 == 0 && (uintptr_t)c.in % 16 == 0;
    auto run = [&](auto kernel, int w) {
        return tsb_launch(ctx, kernel, dim3((unsigned)c.tiles.n, (unsigned)((c.channels + THREADS * w - 1) / (THREADS * w))), dim3(THREADS), 0, st, true, c, ctx->dev_error);
    };
    if (c.taps <= 4) {
        if (f32) return vec ? run(short_conv_kernel<float, 4, 4, RESIDUAL>, 4) : run(short_conv_kernel<float, 1, 4, RESIDUAL>, 1);
        return vec ? run(short_conv_kernel<__nv_bfloat16, 4, 4, RESIDUAL>, 4) : run(short_conv_kernel<__nv_bfloat16, 1, 4, RESIDUAL>, 1);
    }
    return f32 ? run(short_conv_kernel<float, 1, CONV_MAX_TAPS, RESIDUAL>, 1) : run(short_conv_kernel<__nv_bfloat16, 1, CONV_MAX_TAPS, RESIDUAL>, 1);
}

}  // namespace

bool sublayer_end_supported(int d, int groups, int taps) {
    return groups > 0 && d % groups == 0 && taps >= 0 && taps <= CONV_MAX_TAPS && (by_fours(d, groups) || d <= THREADS * MAX_VECS1) && d / 4 + groups <= 10000;
}
int sublayer_rows_per_tile(const tsb_ctx* ctx, int rows) {
    const int sms = ctx->sm_count > 0 ? ctx->sm_count : 148;
    if (rows <= 2 * sms) return 1;
    return rows <= 8 * sms ? 4 : std::max(8, std::min(16, (rows + sms - 1) / sms));  // one CTA per SM where that is enough
}

cudaError_t launch_sublayer_end(tsb_ctx* ctx, cudaStream_t st, bool f32, const SublayerEnd& s) {
    auto run = [&](const SublayerEnd& v) { return f32 ? launch_end_of<float>(ctx, st, v) : launch_end_of<__nv_bfloat16>(ctx, st, v); };
    if (s.taps == 0 || !s.experts || s.n_rows <= 2 * ctx->sm_count) return run(s);
    // many sums of experts: a CTA per row, then the convolution, instead of runs of rows that make the rows before them again
    SublayerEnd sum = s;
    sum.taps = 0, sum.tiles = RowTiles::uniform(s.n_rows, 1, 1);
    if (cudaError_t e = run(sum); e != cudaSuccess) return e;
    ShortConv c;
    c.in = s.x_out, c.in_stride = s.d, c.out = s.out, c.out_stride = s.out_stride, c.channels = s.d, c.taps = s.taps, c.w = s.taps_w, c.ring = s.ring;
    c.use_before = s.use_before, c.rows = s.rows, c.n_rows = s.n_rows, c.tiles = s.tiles;
    return launch_conv<true>(ctx, st, f32, c);
}

cudaError_t launch_rings_before(tsb_ctx* ctx, cudaStream_t st, const RowRing* rings_dev, int n, const tsb_row_desc* rows_dev, const RowTiles& portions) {
    return tsb_launch(ctx, rings_before_kernel, dim3((unsigned)portions.n, (unsigned)n), dim3(THREADS), 0, st, true, rings_dev, rows_dev, portions);
}

cudaError_t launch_group_norm_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* weight, int groups, float eps, const int32_t* want_dev,
                                   int want_first, int want_step, int n, void* out, int64_t out_stride) {
    return f32 ? launch_norm_of(ctx, st, x, d, weight, groups, eps, want_dev, want_first, want_step, n, (float*)out, out_stride)
               : launch_norm_of(ctx, st, x, d, weight, groups, eps, want_dev, want_first, want_step, n, (__nv_bfloat16*)out, out_stride);
}

cudaError_t launch_projection_norms(tsb_ctx* ctx, cudaStream_t st, bool f32, const ProjectionNorms& p, int rows) {
    auto run = [&](auto kernel) { return tsb_launch(ctx, kernel, dim3((unsigned)rows, 2), dim3(THREADS), 0, st, true, p, ctx->dev_error); };
    const bool vec = p.width % 4 == 0 && p.raw_stride % 4 == 0 && p.q_stride % 4 == 0 && p.q_step % 4 == 0 && p.keys.head_step % 4 == 0;
    if (f32) return vec ? run(projection_norms_kernel<float, 4>) : run(projection_norms_kernel<float, 1>);
    return vec ? run(projection_norms_kernel<__nv_bfloat16, 4>) : run(projection_norms_kernel<__nv_bfloat16, 1>);
}

cudaError_t launch_short_conv(tsb_ctx* ctx, cudaStream_t st, bool f32, const ShortConv& c) { return launch_conv<false>(ctx, st, f32, c); }

cudaError_t launch_gated_norm(tsb_ctx* ctx, cudaStream_t st, bool f32, const GatedNorm& g, int rows) {
    const int gw = g.width / g.groups;
    const bool vec = gw % 4 == 0 && g.weight_n % 4 == 0 && g.o_stride % 4 == 0 && g.out_stride % 4 == 0 && g.gate_stride % 4 == 0 &&
                     (uintptr_t)g.pre_gate % 16 == 0 && (uintptr_t)g.post_gate % 16 == 0 && (uintptr_t)g.out % 16 == 0;
    auto run = [&](auto kernel, int w, SmemOptIn& configured) {
        const size_t smem = ((size_t)g.width + g.width / w + g.groups) * sizeof(float);
        if (smem > 48 * 1024)
            if (cudaError_t e = tsb_opt_in_smem(ctx, kernel, 200 * 1024, configured); e != cudaSuccess) return e;
        return tsb_launch(ctx, kernel, dim3((unsigned)rows), dim3(THREADS), smem, st, true, g);
    };
    static SmemOptIn configured[4];
    if (f32) return vec ? run(gated_norm_kernel<float, 4>, 4, configured[0]) : run(gated_norm_kernel<float, 1>, 1, configured[1]);
    return vec ? run(gated_norm_kernel<__nv_bfloat16, 4>, 4, configured[2]) : run(gated_norm_kernel<__nv_bfloat16, 1>, 1, configured[3]);
}
