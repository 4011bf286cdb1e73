// Matrix products with plain (unquantised) weights, bfloat16 or f32, and the epilogues of the plain-weight decoder
// layers.  y[t, n] = sum_k W[n, k] * x[t, k].
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"
#include "experts.cuh"
#include "kv.cuh"

// Weight matrices are packed for the kernels when they are uploaded: rows padded with zero rows to a multiple of
// PLAIN_ROW_PAD, columns with zero columns to a multiple of PLAIN_COL_PAD (activations have the same row stride and
// zeros there).  Gate and up rows of a feed-forward are interleaved in groups of eight - gate 8i .. 8i + 7, then up
// 8i .. 8i + 7 - so that the two halves of a pair meet in one tile, and in one thread of an mma fragment.
constexpr int PLAIN_ROW_PAD = 128;
constexpr int PLAIN_COL_PAD = 64;
inline int64_t plain_pad(int64_t n, int64_t to) { return (n + to - 1) / to * to; }

enum PlainEpiKind {
    PLAIN_STORE = 0,  // y[t, n] = acc, through cap * tanh(acc / cap) when cap > 0
    PLAIN_ADD = 1,    // y[t, n] = alpha * y[t, n] + beta * acc  (the residual stream)
    PLAIN_MIXER = 2,  // by row of the matrix: segments with destinations of their own, then pairs of rows (gate and up of a
                      // feed-forward as act(gate) * up, or the two coordinates of a rotation)
};
// Where the rows of a segment go.
enum PlainSegKind {
    PLAIN_SEG_TYPED = 0,  // an activation buffer of the compute type
    PLAIN_SEG_F32 = 1,    // an f32 buffer
    PLAIN_SEG_CACHE = 2,  // the cache row of the token
};
// Rows [end of the segment before, end) in groups of `per`, of which the first `valid` are kept: row i of group g lands at
// element g * step + i of the token's row, which starts at p + t * stride (or, in the cache, `stride` elements into its row).
struct PlainSeg {
    int end = 0, kind = PLAIN_SEG_TYPED;
    int per = 0x7fffffff, valid = 0x7fffffff, step = 0;
    void* p = nullptr;
    int64_t stride = 0;
    const void* gate = nullptr;  // PLAIN_SEG_TYPED: times sigmoid of element g * gate_step + i of row t of this buffer (compute type)
    int64_t gate_stride = 0;
    int gate_step = 0;
    int act = -1;                // PLAIN_SEG_TYPED: a PlainAct of the row's own number (a feed-forward without gates); -1: none
};
constexpr int PLAIN_SEGS = 6;
// Pairs (u, v) as coordinates i and i + half of a rotated part: u c - v s and v c + u s with (c, s) of the token's position.
// Pair p belongs to head p / half; heads below n_heads are queries, the one behind them the key.
struct PlainRotate {
    int half = 0, n_heads = 0;           // half 0: no rotation
    const float2* table = nullptr;       // [t, half]
    void* q[2] = {nullptr, nullptr};     // one or two query buffers: element (head * q_step + q_off) of row t
    int64_t q_stride[2] = {0, 0};
    int q_step[2] = {0, 0}, q_off[2] = {0, 0};
    int key_off = 0;                     // the key's elements start here in the cache row
};
enum PlainAct { PLAIN_GELU_TANH = 0, PLAIN_SILU = 1, PLAIN_RELU2 = 2 };  // RELU2: max(z, 0)^2

struct PlainEpi {
    int kind = PLAIN_STORE;
    int n_valid = 0;       // PLAIN_STORE / PLAIN_ADD: rows of the matrix that have an output column
    float* y = nullptr;
    int64_t y_stride = 0;
    float cap = 0.f, alpha = 1.f, beta = 1.f;
    // PLAIN_MIXER
    PlainSeg seg[PLAIN_SEGS];
    int n_seg = 0;
    const float* bias = nullptr;  // per row of the matrix, added to the rows of segments; null: none
    KeyView keys{};
    const tsb_row_desc* rows = nullptr;
    PlainRotate rot;             // half > 0: the pairs are rotated coordinates
    int pair_row0 = 0x7fffffff;  // the matrix row where the interleaved pairs start (a multiple of PLAIN_ROW_PAD)
    int n_pairs = 0, act = PLAIN_GELU_TANH;
    void* a = nullptr;      // [t, n_pairs], the compute type
    int64_t a_stride = 0;
};

struct PlainMat {
    void* data = nullptr;     // bfloat16 or f32
    int64_t rows = 0, cols = 0;  // padded
    // A block-diagonal product: rows of group g (group_rows each, a multiple of PLAIN_ROW_PAD) multiply the columns of x from
    // g * group_cols on.  0: every row multiplies the same columns.
    int group_rows = 0, group_cols = 0;
};

// A product per expert: the matrix holds n matrices of w.rows rows one after another, and the slots of an expert (experts.cuh) multiply its
// own.  Output rows are slots.
struct PlainExperts {
    int n = 0, slots = 0;
    const int32_t* first = nullptr;      // [n + 1]
    const int32_t* token_of = nullptr;   // row of x of a slot; null: x has a row per slot
    const ExpertChunk* chunks = nullptr;
    const int32_t* n_chunks = nullptr;
    int chunk_slots = 0;
};

// Split sums of products with few row tiles: tickets, then f32 tiles.
size_t plain_gemm_workspace_bytes(const tsb_ctx* ctx);
// Rows of the matrix below epi.pair_row0 multiply x, the others x2; both have x_rows allocated rows of x_stride elements
// (x_rows * x_stride elements are readable, and finite rows past `tokens` are not needed).
cudaError_t launch_plain_gemm(tsb_ctx* ctx, cudaStream_t st, bool f32, const PlainMat& w, const void* x, const void* x2, int64_t x_stride, int x_rows,
                              int tokens, const PlainEpi& epi, void* workspace);
// Slots by expert; x_rows, x_stride as above, epi.kind PLAIN_MIXER.  tensor: on the tensor-memory kernel (bfloat16, x by slots); else chunks
// of at most EXPERT_CHUNK_FEW (bfloat16) or EXPERT_CHUNK_F32 slots.
constexpr int EXPERT_CHUNK_FEW = 16, EXPERT_CHUNK_F32 = 64;
cudaError_t launch_plain_gemm_experts(tsb_ctx* ctx, cudaStream_t st, bool f32, bool tensor, const PlainMat& w, const void* x, int64_t x_stride, int x_rows,
                                      const PlainExperts& ex, const PlainEpi& epi);
