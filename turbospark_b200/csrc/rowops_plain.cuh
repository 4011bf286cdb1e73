// Row operators of the plain-weight decoders: f32 residual stream, activations in the compute type.
#pragma once
#include "common.cuh"

// Rows of the stream's token shift: the normed row of every position, kept for the last ring - 1 rows of a stream.
// [layer][stream][ring][width] f32; position p sits in slot p & (ring - 1).
struct ShiftState {
    float* ring = nullptr;
    float* before = nullptr;  // [layer][stream][width]: copies of the rows before a pass whose portions may overwrite them
    int width = 0, ring_rows = 0, n_streams = 0;
};

// x[r, :] = embedding row of tokens[r * token_stride] (f32 or bfloat16 table [vocab, d])
cudaError_t launch_plain_embed(tsb_ctx* ctx, cudaStream_t st, bool f32, const void* table, int vocab, int d, const int32_t* tokens, int token_stride,
                               int rows, float* x);
// One layer's input: h = x * gain / sqrt(mean(x^2) + eps) in f32.  h_out (compute type, may be null) receives h; mix_out
// receives h + (h' - h) * mu with h' the row before (the pass's own, or the stream's state; zero at position 0), or h
// itself when mu is null.  The state keeps the rows' h.  x2_stride is the row stride of both outputs.
cudaError_t launch_norm_shift(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* gain, float eps, const float* mu,
                              const tsb_row_desc* rows_dev, int rows, ShiftState state, int layer, bool use_before, void* mix_out, void* h_out,
                              int64_t out_stride);
// state.before[layer][stream] = the row before each listed row's portion (rows with slot 0), every layer
cudaError_t launch_shift_before(tsb_ctx* ctx, cudaStream_t st, ShiftState state, int layers, const tsb_row_desc* rows_dev, int rows);
// out[i, :] = norm of x row want(i): want_dev[i], or i * want_step + want_first when want_dev is null
cudaError_t launch_norm_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* gain, float eps, const int32_t* want_dev,
                             int want_first, int want_step, int n, void* out, int64_t out_stride);
