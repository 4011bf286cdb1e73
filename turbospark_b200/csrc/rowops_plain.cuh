// Row operators of the plain-weight decoders: f32 residual stream, activations in the compute type.
#pragma once
#include "common.cuh"
#include "kv.cuh"

// Rows of the stream's token shift: the normed row of every position, kept for the last ring - 1 rows of a stream.
// [layer][stream][ring][width] f32; position p sits in slot p & (ring - 1).
struct ShiftState {
    float* ring = nullptr;
    float* before = nullptr;  // [layer][stream][width]: copies of the rows before a pass whose portions may overwrite them
    int width = 0, ring_rows = 0, n_streams = 0;
};

// x[r, :] = scale * embedding row of tokens[r * token_stride] (f32 or bfloat16 table [vocab, d]); out (may be null) receives
// it in the compute type too
cudaError_t launch_plain_embed(tsb_ctx* ctx, cudaStream_t st, bool f32, const void* table, int vocab, int d, const int32_t* tokens, int token_stride,
                               int rows, float scale, float* x, void* out, int64_t out_stride);
// One layer's input: h = x * gain / sqrt(mean(x^2) + eps) in f32.  h_out (compute type, may be null) receives h; mix_out
// receives h + (h' - h) * mu with h' the row before (the pass's own, or the stream's state; zero at position 0), or h
// itself when mu is null.  The state keeps the rows' h.  x2_stride is the row stride of both outputs.
cudaError_t launch_norm_shift(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* gain, float eps, const float* mu,
                              const tsb_row_desc* rows_dev, int rows, ShiftState state, int layer, bool use_before, void* mix_out, void* h_out,
                              int64_t out_stride);
// state.before[layer][stream] = the row before each listed row's portion (rows with slot 0), every layer
cudaError_t launch_shift_before(tsb_ctx* ctx, cudaStream_t st, ShiftState state, int layers, const tsb_row_desc* rows_dev, int rows);
// out[i, :] = norm of x row want(i): want_dev[i], or i * want_step + want_first when want_dev is null.  weight [d]: a gain per
// coordinate instead of the one of `gain`.
cudaError_t launch_norm_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* gain, const float* weight, float eps,
                             const int32_t* want_dev, int want_first, int want_step, int n, void* out, int64_t out_stride);
// Norm after the sum, in place: x[r, :] = x * weight / sqrt(mean(x^2) + eps) in f32, and in the compute type to out.
cudaError_t launch_post_norm(tsb_ctx* ctx, cudaStream_t st, bool f32, float* x, int d, const float* weight, float eps, int rows, void* out,
                             int64_t out_stride);
// The same without rewriting x: the input of a pre-norm sublayer.
cudaError_t launch_pre_norm(tsb_ctx* ctx, cudaStream_t st, bool f32, const float* x, int d, const float* weight, float eps, int rows, void* out,
                            int64_t out_stride);

// Norms over the heads of a projection: raw [rows, raw_stride] f32 holds n_q heads of `width` numbers, then n_k such heads.
// Each is normed over its width with the weight of its kind; queries are scaled by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1)
// at position p (temp_every 0: not) and stored to q at (head * q_step) with zeros up to q_width; keys go to the token's cache row
// at (head * keys.head_step).  n_q = 0, n_k = 1 is the norm of a latent.  With `rot`, columns 2 i and 2 i + 1 of a normed head are turned by
// (cos, sin) of [rows, rot_half].  n_v heads of v_width numbers behind the keys are values: not normed, turned by `turn`, stored keys.value_off
// elements into the cache's heads.  pool > 0: the block that ends right before a portion gets its mean (see BlockMeans; its rows are all of earlier passes).
struct HeadNorms {
    const float* raw = nullptr;
    int64_t raw_stride = 0;
    int n_q = 0, n_k = 0, width = 0;
    const float *q_weight = nullptr, *k_weight = nullptr;
    float eps = 0.f;
    float temp_coef = 0.f;
    int temp_every = 0;
    void* q = nullptr;
    int64_t q_stride = 0;
    int q_step = 0, q_width = 0;
    const float2 *rot = nullptr, *turn = nullptr;
    int rot_half = 0, turn_half = 0, n_v = 0, v_width = 0;
    KeyView keys{}, pooled{};
    int pool = 0;
    const tsb_row_desc* rows = nullptr;
};
cudaError_t launch_head_norms(tsb_ctx* ctx, cudaStream_t st, bool f32, const HeadNorms& h, int rows);

// Rows of blocks (KeyLayerShape::pool): where a row of the pass is the last position of a block of `pool`, the block's row becomes the mean of the cache's
// rows at its positions - all of them written before - summed in f32 in their order.
struct BlockMeans {
    KeyView keys{}, pooled{};
    int pool = 0;
    const tsb_row_desc* rows = nullptr;
};
cudaError_t launch_block_means(tsb_ctx* ctx, cudaStream_t st, bool f32, const BlockMeans& b, int rows);

// table[r, i] = magnitude * (cos, sin)(position of row r * freq[i]), i below half; the product is reduced to one turn in double
cudaError_t launch_rotary_table(tsb_ctx* ctx, cudaStream_t st, const double* freq, int half, float magnitude, const tsb_row_desc* rows_dev, int rows,
                                float2* table);

// Cached latent rows of whole streams, for their expansion to keys and values (bfloat16).  Stream i of the list (first row of
// its portion in the pass, rows of the portion, first page of its place) occupies consecutive pages of `wide`, a cache view whose
// page table [max_seqs][max_pages_per_seq] is written here.  Per position: the latent row to latents, and to every head of the
// wide row the rotated key part at key_off, zeros up to the head's key width.
struct ExpandStream {
    int32_t first_row, n_rows, first_page;
};
struct LatentGather {
    KeyView cache{}, wide{};
    int32_t* wide_table = nullptr;
    void* latents = nullptr;
    int kv_rank = 0, rot_dim = 0, key_off = 0;
    const tsb_row_desc* rows = nullptr;
    const ExpandStream* streams = nullptr;
};
cudaError_t launch_latent_gather(tsb_ctx* ctx, cudaStream_t st, const LatentGather& g, int n_streams, int max_len);
