// Shared by the sliding-window attention kernels: score arithmetic helpers and the launch description.
#pragma once
#include "attention_window.cuh"

namespace {

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float lg2(float x) {
    float y;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// What a head's sum of weighted values is multiplied by (bfloat16 kernels: m and l in base 2): one over the sum of the weights -
// the sink's among them - times the head's gate.
__device__ __forceinline__ float head_factor(const WindowAttn& a, int row, int head, float m, float l) {
    if (a.sink) l += ex2(a.sink[head] * 1.4426950408889634f - (m == -INFINITY ? 0.f : m));
    float f = l > 0.f ? 1.f / l : 0.f;
    if (a.gate) f *= sigmoid(a.gate[(int64_t)row * a.n_q_heads + head]);
    return f * a.out_scale;
}
// the earliest position that a query at `pos` sees
__device__ __forceinline__ int first_visible(const WindowAttn& a, int pos) {
    return a.window > 0 ? max(0, pos - a.window + 1) : a.chunk > 0 ? pos - pos % a.chunk : 0;
}
// How much of the prefix - kept positions, or blocks - a query at `pos` sees: all of it that lies before the window.
__host__ __device__ __forceinline__ int prefix_len(const WindowAttn& a, int pos) {
    const int before = pos - a.window + 1;  // positions before the window
    return before <= 0 ? 0 : a.pool > 0 ? before / a.pool : before < a.keep ? before : a.keep;
}
// Row i of the prefix, or position i of the stream; nullptr outside the reserved pages.
__device__ __forceinline__ const __nv_bfloat16* run_row(const WindowAttn& a, bool prefix, int seq, int i) {
    const bool pooled = prefix && a.pool > 0;
    const int shift = pooled ? a.pooled.page_shift : a.keys.page_shift, lp = i >> shift;
    if (i < 0 || lp >= a.keys.max_pages_per_seq) return nullptr;
    const int page = a.keys.page_table[(size_t)seq * a.keys.max_pages_per_seq + lp];
    if (page < 0) return nullptr;
    return reinterpret_cast<const __nv_bfloat16*>(pooled ? a.pooled.base : a.keys.base) + (((int64_t)page << shift) + (i & ((1 << shift) - 1))) * a.keys.row;
}
// The output columns c and c + 1 (c even) of a row, turned back to the row's position.
__device__ __forceinline__ void turn_back(const WindowAttn& a, int row, int c, float& u, float& v) {
    if (c >= 2 * a.turn_half) return;
    const float2 t = a.turn[(int64_t)row * a.turn_half + (c >> 1)];
    const float x = fmaf(u, t.x, v * t.y);
    v = fmaf(v, t.x, -u * t.y), u = x;
}
// how many positions, itself included, a query at `pos` sees at most (a number no distance reaches: all of them)
__device__ __forceinline__ float visible_span(const WindowAttn& a, int pos) {
    return a.window > 0 ? (float)a.window : a.chunk > 0 ? (float)(pos % a.chunk + 1) : 3e38f;
}
// the gate of value column c, and of four from c (a multiple of four) on
__device__ __forceinline__ const __nv_bfloat16* value_gate_at(const WindowAttn& a, int row, int head, int c) {
    return static_cast<const __nv_bfloat16*>(a.value_gate) + (int64_t)row * a.value_gate_stride + (int64_t)head * (a.value_dim > 0 ? a.value_dim : a.keys.head_dim) + c;
}
__device__ __forceinline__ float value_gate(const WindowAttn& a, int row, int head, int c) { return sigmoid(__bfloat162float(*value_gate_at(a, row, head, c))); }
__device__ __forceinline__ void value_gates(const WindowAttn& a, int row, int head, int c, float4& v) {
    const uint2 w = *reinterpret_cast<const uint2*>(value_gate_at(a, row, head, c));
    v.x *= sigmoid(__uint_as_float(w.x << 16)), v.y *= sigmoid(__uint_as_float(w.x & 0xFFFF0000u));
    v.z *= sigmoid(__uint_as_float(w.y << 16)), v.w *= sigmoid(__uint_as_float(w.y & 0xFFFF0000u));
}

__device__ __forceinline__ float max3(float a, float b, float c) {
    float d;
    asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
    return d;
}

// Two f32 lanes per instruction.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;"
        : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)),
          "l"(reinterpret_cast<const unsigned long long&>(c)));
    return d;
}
__device__ __forceinline__ float2 add2(float2 a, float2 b) {
    float2 d;
    asm("add.rn.f32x2 %0, %1, %2;"
        : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)));
    return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("mul.rn.f32x2 %0, %1, %2;"
        : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)));
    return d;
}
__device__ __forceinline__ float2 both(float x) { return make_float2(x, x); }

// Within |y| <= TANH_SMALL, tanh(y) / y is a cubic in y^2, interpolated at the Chebyshev nodes of the range: 1.1e-8 off at most, 6e-8 with
// f32 rounding.  Scores well inside the cap - the usual case - then need no special-function instruction but the softmax's own.
constexpr float TANH_SMALL = 0.3f;
// Constants of the way from a raw score x = q . k to a base-2 logit: c_out tanh(x scale / cap), or x s_in without a cap.
struct ScoreConst {
    float s_in, c_out, small, k0, k1, k2, k3;
    __device__ __forceinline__ explicit ScoreConst(const WindowAttn& a) {
        constexpr float LOG2E = 1.4426950408889634f;
        const bool capped = a.cap > 0.f;
        s_in = capped ? a.scale / a.cap * (2.f * LOG2E) : a.scale * LOG2E;  // capped: the exponent of e^(2 y) in base 2
        c_out = a.cap * LOG2E;
        // the polynomial in x: x (k0 + k1 x^2 + ...)
        const float y = capped ? a.scale / a.cap : 0.f, y2 = y * y;
        small = capped ? TANH_SMALL / fabsf(y) : 0.f;
        const float k = c_out * y;
        k0 = k * 0.99999998957f, k1 = k * y2 * -0.33332962017f, k2 = k * y2 * y2 * 0.13312577658f, k3 = k * y2 * y2 * y2 * -0.05022099099f;
    }
    // what a pair of raw scores inside the range is multiplied by
    __device__ __forceinline__ float2 factor(float2 x) const;
};

inline bool has_prefix(const WindowAttn& a) { return a.keep > 0 || a.pool > 0; }

__device__ __forceinline__ float2 ScoreConst::factor(float2 x) const {
    const float2 z = mul2(x, x);
    return fma2(z, fma2(z, fma2(z, both(k3), both(k2)), both(k1)), both(k0));
}

constexpr int WATTN_TICKETS = 16384;
constexpr int WATTN_MAX_SPLITS = 64;

}  // namespace

struct WattnLaunch {
    const AttnTile* tiles;  // null: a uniform pass
    int n_tiles, tiles_per_group, rows_per_seq, rows_per_tile, max_len;
};
// Scratch of cut tiles: tickets, then (m, l) of every query slot, then the slots' sums.
struct WattnScratch {
    uint32_t* tickets;
    float2* ml;
    float* o;
};
inline size_t wattn_part_queries(const tsb_ctx* ctx) { return (size_t)4 * (ctx->sm_count > 0 ? ctx->sm_count : 148) * WATTN_SMALL_Q; }
inline WattnScratch wattn_scratch(const tsb_ctx* ctx, void* p) {
    WattnScratch s;
    s.tickets = static_cast<uint32_t*>(p);
    s.ml = reinterpret_cast<float2*>(s.tickets + WATTN_TICKETS);
    s.o = reinterpret_cast<float*>(s.ml + wattn_part_queries(ctx));
    return s;
}
// How many runs the key tiles of a launch are cut into: the number whose waves come out most even.  base: CTAs of an uncut
// launch; a CTA costs its key tiles plus about three tiles' time of fixed work, a cut tile also the merge of its runs.
inline int wattn_splits(const tsb_ctx* ctx, int window, const WattnLaunch& l, int tile_tokens, int queries_per_cta, int ctas_per_sm, int base,
                        size_t part_queries, int prefix = 0) {
    const int sms = ctx->sm_count > 0 ? ctx->sm_count : 148;
    const int span = window > 0 && window + l.rows_per_tile < l.max_len ? window + l.rows_per_tile : l.max_len;
    const int key_tiles = (span + tile_tokens - 1) / tile_tokens + (window > 0 ? 1 : 0) + (prefix + tile_tokens - 1) / tile_tokens;
    int splits = 1;
    float best = 1e30f;
    for (int s = 1; s <= WATTN_MAX_SPLITS && s <= (key_tiles + 1) / 2; s++) {
        if (s > 1 && ((int64_t)base * s * queries_per_cta > (int64_t)part_queries || base > WATTN_TICKETS)) break;
        const int waves = (base * s + ctas_per_sm * sms - 1) / (ctas_per_sm * sms);
        const float cost = (float)waves * ((float)((key_tiles + s - 1) / s) + 3.f) + (s > 1 ? 3.f + 0.1f * (float)s : 0.f);
        if (cost < best - 1e-3f) best = cost, splits = s;
    }
    return splits;
}
inline int wattn_splits(const tsb_ctx* ctx, const WindowAttn& a, const WattnLaunch& l, int tile_tokens, int queries_per_cta, int ctas_per_sm) {
    return wattn_splits(ctx, a.window > 0 ? a.window : a.chunk, l, tile_tokens, queries_per_cta, ctas_per_sm, l.n_tiles * a.keys.kv_heads, wattn_part_queries(ctx),
                        a.window > 0 && has_prefix(a) ? prefix_len(a, l.max_len - 1) : 0);
}

// Adds the runs of cut tiles, in order, and writes the finished rows.  A tile has `slots` query slots per run: row r of the
// tile and head h sit in slot (r / R) * 128 + (r % R) * group + h with R = 128 / group.
cudaError_t launch_window_attn_merge(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int splits, int slots, const WattnScratch& sc);

// The tcgen05 kernels for many queries (attention_window_tc.cuh): head sizes 64 and 128, with a distance bias up to eight heads
// per key head.
bool wattn_tc_supported(int head_dim, int group, bool biased);
cudaError_t launch_window_attn_tc(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch);
// The kernels for caches with values of their own (attention_kv.cu, attention_kv_tc.cu).
cudaError_t launch_kv_attn_small(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int queries, void* scratch);
cudaError_t launch_kv_attn_large(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch);
cudaError_t launch_kv_attn_tc(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch);
// The same with a prefix before the window (attention_prefix.cu, attention_prefix_tc.cu).
cudaError_t launch_prefix_attn_small(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int queries, void* scratch);
cudaError_t launch_prefix_attn_large(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch);
cudaError_t launch_prefix_attn_tc(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch);
