// Attention over latent rows: every query head reads the same paged row - the latent, which is also its value, and behind it a
// rotated key part - with a per-head sink (optional).  Queries and outputs live in the latent's space: the heads' own key and
// value matrices have been multiplied into the query, and are applied to the output, by the caller.
#pragma once
#include "attention_window.cuh"

struct LatentAttn {
    KeyView keys{};           // one head of head_dim columns, the first value_dim of them the value
    const void* q = nullptr;  // [rows, n_heads, head_dim] bfloat16
    int64_t q_stride = 0;
    void* out = nullptr;      // [rows, n_heads, value_dim] bfloat16
    int64_t out_stride = 0;
    const tsb_row_desc* rows = nullptr;
    int n_heads = 0, value_dim = 0;
    float scale = 1.f;
    const float* sink = nullptr;
};

// The columns the kernels work on for a latent of kv_rank numbers and a rotated part of rot_dim: false if there is no kernel.
bool latent_attn_dims(int kv_rank, int rot_dim, int* key_dim, int* value_dim);
// A query tile: rows of one stream times heads.  `rows`: how many rows a list's tiles may have.
struct LatentTiling {
    int queries, heads, rows;  // queries of a tile, heads of it, rows of it
};
// most_rows: the longest portion of the launch, n_rows: rows of all portions, max_len: the longest visible context
LatentTiling latent_attn_tiling(const tsb_ctx* ctx, int n_heads, int most_rows, int n_rows, int max_len);
// `large` is not used: every tile of b.small has at most the tiling's rows
cudaError_t launch_latent_attn(tsb_ctx* ctx, cudaStream_t st, const LatentAttn& a, const AttnBatch& b, const LatentTiling& t, void* scratch);
