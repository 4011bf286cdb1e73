// Matrix products with plain (unquantised) weights, bfloat16 or f32, and the epilogues of the plain-weight decoder
// layers.  y[t, n] = sum_k W[n, k] * x[t, k].
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"
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
    PLAIN_ADD = 1,    // y[t, n] += acc  (the residual stream)
    PLAIN_MIXER = 2,  // the projections of a layer, by row: queries, keys straight into the cache, head gates, then
                      // gate / up pairs of the feed-forward as act(gate) * up
};
enum PlainAct { PLAIN_GELU_TANH = 0, PLAIN_SILU = 1 };

struct PlainEpi {
    int kind = PLAIN_STORE;
    int n_valid = 0;       // PLAIN_STORE / PLAIN_ADD: rows of the matrix that have an output column
    float* y = nullptr;
    int64_t y_stride = 0;
    float cap = 0.f;
    // PLAIN_MIXER
    void* q = nullptr;     // [t, q_rows], the compute type
    int64_t q_stride = 0;
    int q_rows = 0, k_rows = 0, gate_rows = 0;
    KeyView keys{};
    const tsb_row_desc* rows = nullptr;
    float* gate = nullptr;  // [t, gate_rows]: the gates' pre-activations
    int pair_row0 = 0x7fffffff;  // the matrix row where the interleaved pairs start (a multiple of PLAIN_ROW_PAD)
    int n_pairs = 0, act = PLAIN_GELU_TANH;
    void* a = nullptr;      // [t, n_pairs], the compute type
    int64_t a_stride = 0;
};

struct PlainMat {
    void* data = nullptr;     // bfloat16 or f32
    int64_t rows = 0, cols = 0;  // padded
};

// Split sums of products with few row tiles: tickets, then f32 tiles.
size_t plain_gemm_workspace_bytes(const tsb_ctx* ctx);
// Rows of the matrix below epi.pair_row0 multiply x, the others x2; both have x_rows allocated rows of x_stride elements
// (x_rows * x_stride elements are readable, and finite rows past `tokens` are not needed).
cudaError_t launch_plain_gemm(tsb_ctx* ctx, cudaStream_t st, bool f32, const PlainMat& w, const void* x, const void* x2, int64_t x_stride, int x_rows,
                              int tokens, const PlainEpi& epi, void* workspace);
