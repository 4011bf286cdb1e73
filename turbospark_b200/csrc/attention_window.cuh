// Attention over a plain paged cache - a layer's values are its keys, or stand behind them - with a sliding window
// or a chunk mask, a prefix that stays visible beside the window (kept first tokens, or means of the blocks before it), a soft cap on the
// scores, a per-head logarithmic or linear distance bias, a per-head sink, values that turn with their position, and output gates per
// head or per value column - each of them optional.
#pragma once
#include <cuda_bf16.h>

#include "kv.cuh"

struct WindowAttn {
    KeyView keys{};
    const void* q = nullptr;  // [rows, n_q_heads * keys.head_dim], the compute type
    int64_t q_stride = 0;
    const float* gate = nullptr;  // [rows, n_q_heads]: a head's output is multiplied by sigmoid(gate); null: no gate
    void* out = nullptr;      // [rows, n_q_heads * keys.head_dim], the compute type
    int64_t out_stride = 0;
    const tsb_row_desc* rows = nullptr;  // position base + slot; the rows of a stream are consecutive
    int n_q_heads = 0;
    float scale = 1.f;        // score = (q . k) * scale
    float cap = 0.f;          // > 0: score <- cap * tanh(score / cap)
    const float *r1 = nullptr, *r2 = nullptr;  // per head: score <- score - r1 * ln(1 + r2 * distance); null: no bias
    const float* slopes = nullptr;             // per head: score <- score - slope * distance; null: no such bias (not with r1)
    int chunk = 0;            // > 0: a query sees the positions of its own chunk (counted from position 0) up to itself; not with a window
    int window = 0;           // a query sees itself and the window - 1 positions before it; 0: every earlier position
    // What stays visible before the window (window > 0, values of their own, no distance bias): the stream's first `keep` positions, or - pool > 0 -
    // a row of `pooled` for each block of `pool` positions that lies wholly before the window.
    int keep = 0, pool = 0;
    KeyView pooled{};             // shaped like keys but for its pages
    const float* sink = nullptr;  // per head: exp(sink) joins the softmax's denominator
    // [rows, n_q_heads * value columns], the compute type: a head's output is multiplied by the sigmoid, column by column
    const void* value_gate = nullptr;
    int64_t value_gate_stride = 0;
    // values that turn with their position: (cos, sin) of [rows, turn_half] at the rows' positions; columns 2 m and 2 m + 1 of a head's output
    // are turned back by them, before any gate
    const float2* turn = nullptr;
    int turn_half = 0;
    float out_scale = 1.f;    // of the heads' outputs
    int value_dim = 0;        // value columns (the heads of out and value_gate are as wide); 0: as many as a key has
};

// A query tile: consecutive rows of one stream times the query heads of one key head.
struct AttnTile {
    int32_t row_first, n_rows;
};
constexpr int WATTN_SMALL_Q = 64;   // queries (rows x heads per key head) of a stream up to which the few-query kernel takes them
constexpr int WATTN_LARGE_Q = 128;  // queries per tile of the many-query kernels (a tcgen05 CTA takes two such tiles)
int wattn_rows_per_tile(int head_dim, int group, bool biased);  // rows of a tile in the many-query kernel that takes this geometry

// Where the query tiles of a pass come from: a uniform pass (rows_per_seq rows of every stream) or device lists made for
// the layer's group size by wattn_make_tiles.
struct AttnBatch {
    int rows = 0, rows_per_seq = 0;
    const AttnTile *small = nullptr, *large = nullptr;  // device
    int n_small = 0, n_large = 0, small_queries = 0;    // small_queries: most queries of a small tile
    int max_len = 0;                                    // longest visible context (sizes the splits)
};
size_t wattn_scratch_bytes(const tsb_ctx* ctx);  // zeroed once by the owner; the kernels leave its tickets at zero
bool wattn_supported(int head_dim, int group, bool f32);
int wattn_pad_dim(int head_dim, bool f32);       // the head size the kernels work on (zero columns behind the real ones); 0: too large
// The many-query kernel for keys and values of different widths: every query head has a key head of its own; the `large` tiles
// of a list have at most WATTN_WIDE_ROWS rows.
constexpr int WATTN_WIDE_ROWS = 2 * WATTN_LARGE_Q;
bool wattn_wide_supported(int key_dim, int value_dim);
cudaError_t launch_window_attn_wide(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const AttnBatch& b, void* scratch);
cudaError_t launch_window_attn(tsb_ctx* ctx, cudaStream_t st, bool f32, const WindowAttn& a, const AttnBatch& b, void* scratch);
