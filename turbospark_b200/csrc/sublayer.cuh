// Row operators around the sublayers of output-norm layers: f32 residual stream, activations in the compute type.
#pragma once
#include "stream_state.cuh"

constexpr int CONV_MAX_TAPS = 8;

// The end of a sublayer and the start of the next.  Per row t of the pass:
//   x_out[t] = x_in[t] + norm(s)          s: the sublayer's output, normed in `groups` equal parts
//   out[t]   = x_out[t] + sum_j taps_w[j] * x_out[t - taps + 1 + j]      (f32, then the compute type; taps 0: nothing is written)
// s is a row of y, or the weighted sum of `top` expert outputs.  With a table, x_out is an embedding row (plus a position's row) instead.
struct SublayerEnd {
    const float* x_in = nullptr;  // [rows, d]; not the memory of x_out
    float* x_out = nullptr;
    int d = 0;
    const float* y = nullptr;     // [rows, d]
    const void* experts = nullptr;  // [slots, expert_stride], the compute type
    int64_t expert_stride = 0;
    const int32_t* slot_of = nullptr;  // [rows, top]
    const float* weight = nullptr;     // [rows, top]
    int top = 0;
    const void *table = nullptr, *positions = nullptr;  // [vocab, d], [n_positions, d] (may be null), the compute type
    const int32_t* tokens = nullptr;
    int token_stride = 1, vocab = 0, n_positions = 0;
    float embed_scale = 1.f;
    const float* norm_w = nullptr;
    int groups = 1;
    float eps = 0.f;
    const float* taps_w = nullptr;  // [taps][d]
    int taps = 0;
    RowRing ring{};                 // x_out of the rows before, keep = taps - 1
    bool use_before = false;
    void* out = nullptr;
    int64_t out_stride = 0;
    const tsb_row_desc* rows = nullptr;
    int n_rows = 0;
    RowTiles tiles{};
};
bool sublayer_end_supported(int d, int groups, int taps);
int sublayer_rows_per_tile(const tsb_ctx* ctx, int rows);  // rows of a tile that suit a pass of so many rows
cudaError_t launch_sublayer_end(tsb_ctx* ctx, cudaStream_t st, bool f32, const SublayerEnd& s);

// Copies of the rows before every portion of the pass, of n rings in device memory, to their `before`.
cudaError_t launch_rings_before(tsb_ctx* ctx, cudaStream_t st, const RowRing* rings_dev, int n, const tsb_row_desc* rows_dev, const RowTiles& portions);

// out[i] = x[want(i)] normed in groups, want(i) as in launch_norm_rows.
cudaError_t launch_group_norm_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* weight, int groups, float eps, const int32_t* want_dev,
                                   int want_first, int want_step, int n, void* out, int64_t out_stride);

// Norms of whole projections: raw [rows, raw_stride] f32 holds n_q heads of `width` numbers, then n_k heads.  All queries of a row are
// normed at once, and all keys; weights [n_q * width] and [n_k * width].  Queries go to q (head * q_step, zeros up to q_step), keys to the
// token's cache row (head * keys.head_step).  With `rot`, columns 2 i and 2 i + 1 of a normed head are turned by (cos, sin) of [rows, rot_half].
struct ProjectionNorms {
    const float* raw = nullptr;
    int64_t raw_stride = 0;
    int n_q = 0, n_k = 0, width = 0;
    const float *q_weight = nullptr, *k_weight = nullptr;
    float eps = 0.f;
    void* q = nullptr;
    int64_t q_stride = 0;
    int q_step = 0;
    const float2* rot = nullptr;
    int rot_half = 0;
    KeyView keys{};
    const tsb_row_desc* rows = nullptr;
};
cudaError_t launch_projection_norms(tsb_ctx* ctx, cudaStream_t st, bool f32, const ProjectionNorms& p, int rows);

// Causal convolution per channel with silu: out[t, c] = silu(bias[c] + sum_j w[j][c] * in[t - taps + 1 + j, c]); the ring holds `in`.
struct ShortConv {
    const void* in = nullptr;  // [rows, in_stride], the compute type
    int64_t in_stride = 0;
    void* out = nullptr;
    int64_t out_stride = 0;
    int channels = 0, taps = 0;
    const float *w = nullptr, *bias = nullptr;  // [taps][channels], [channels]
    RowRing ring{};
    bool use_before = false;
    const tsb_row_desc* rows = nullptr;
    int n_rows = 0;
    RowTiles tiles{};
};
cudaError_t launch_short_conv(tsb_ctx* ctx, cudaStream_t st, bool f32, const ShortConv& c);

// The way from a recurrence's output o [rows, width] f32 to the output projection's input: v = o, times silu(pre_gate); normed in equal
// groups; times weight (repeated every weight_n columns); times sigmoid(post_gate); times scale.
struct GatedNorm {
    const float* o = nullptr;
    int64_t o_stride = 0;
    int width = 0, groups = 1, weight_n = 0;
    const float* weight = nullptr;
    float eps = 0.f, scale = 1.f;
    const void *pre_gate = nullptr, *post_gate = nullptr;  // [rows, gate_stride], the compute type
    int64_t gate_stride = 0;
    void* out = nullptr;
    int64_t out_stride = 0;
};
cudaError_t launch_gated_norm(tsb_ctx* ctx, cudaStream_t st, bool f32, const GatedNorm& g, int rows);
