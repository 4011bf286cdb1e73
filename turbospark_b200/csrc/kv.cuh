// Paged fp16 K/V cache: host-side object and the device-side view kernels use.
#pragma once
#include <vector>

#include "common.cuh"

// What a kernel needs to address a row of the cache.  Pool layout:
// [layer][K|V][page][token_in_page][kv_head][head_dim] f16.
struct KvView {
    __half* pool;
    const int32_t* page_table;  // [max_seqs][max_pages_per_seq], -1 = not reserved
    int layers, kv_heads, head_dim;
    int page_tokens, page_shift;
    int num_pages, max_seqs, max_pages_per_seq;
    int64_t kv_stride;     // elements between the K and V halves of a layer
    int64_t layer_stride;  // elements between layers
};

// One layer of a plain cache: token rows of `row` elements, f32 or bfloat16, [page][token_in_page][row].  A row holds
// kv_heads heads, head_step elements apart; a head's key is head_dim elements from its start, its value starts value_off
// elements behind it:
//   values that are their keys   head_step = head_dim, value_off = 0
//   keys and values              head_step = head_dim + the value's elements, value_off = head_dim
//   latent rows                  one head: the latent, which is also the value, then the rotated key part
// Layers may differ in all of it.
struct KeyView {
    uint8_t* base;
    const int32_t* page_table;
    int kv_heads, head_dim, elem_bytes;
    int row, head_step, value_off;
    int page_shift, page_tokens, num_pages, max_seqs, max_pages_per_seq;
};
struct KeyLayerShape {
    int kv_heads, head_dim;  // no heads: the layer has no rows
    int value_dim; // elements of the value behind every key (0: the values are the keys)
    int source;    // the layer whose rows this one reads (itself: rows of its own)
    int pool = 0;  // > 0: the layer also keeps a row for every block of this many positions
};

struct tsb_kv {
    tsb_ctx* ctx = nullptr;
    KvView view{};                    // page geometry; pool and strides of a key + value cache
    std::vector<KeyView> key_layers;  // not empty: a plain cache (view.pool is then null)
    // Rows of blocks (KeyLayerShape::pool), shaped like the layer's rows: row b of a stream belongs to its positions b pool .. b pool + pool - 1.
    // A page of positions brings room for a page of blocks - page_tokens / pool of them, rounded up to a power of two of at least
    // POOLED_MIN_ROWS - and both go by the same page table.  Layers without have no base.
    std::vector<KeyView> pooled_layers;
    std::vector<int> pool_sizes;  // of the layers; 0: none
    uint8_t* key_pool = nullptr;
    // A model whose rows also need their predecessors' state keeps the last state_ring - 1 rows' worth of it per stream
    // (0: no such state).  state_lo is the oldest position whose state is still there: a cursor may go back to 0 or to
    // state_lo + 1 and later.
    int state_ring = 0;
    std::vector<int64_t> state_lo;
    int32_t* page_table_dev = nullptr;
    std::vector<int32_t> page_table_host;
    std::vector<int32_t> free_pages;
    std::vector<int32_t> pages_of_seq;
    std::vector<int64_t> cursor;
};

constexpr int POOLED_MIN_ROWS = 8;  // a copy box of eight rows fills the 1024 bytes after which a 128-byte swizzle repeats
// A plain cache of n_layers layers with their own head counts and (padded) head sizes.
int32_t kv_create_keys(tsb_ctx* ctx, int n_layers, const KeyLayerShape* shapes, int elem_bytes, int page_tokens, int num_pages, int max_seqs,
                       int max_pages_per_seq, tsb_kv** out);
// Seeded pseudo-random rows [0, tokens) of a stream in every layer of a plain cache (reserves the pages).
int32_t kv_fill_keys(tsb_kv* kv, cudaStream_t st, int32_t seq, int64_t tokens, uint64_t seed);

#ifdef __CUDACC__
// Row of a plain layer at position `pos` of stream `seq`; nullptr outside the reserved pages.
template <typename T>
__device__ __forceinline__ T* key_row(const KeyView& kv, int seq, int pos) {
    const int lp = pos >> kv.page_shift;
    if (pos < 0 || seq < 0 || seq >= kv.max_seqs || lp >= kv.max_pages_per_seq) return nullptr;
    const int page = kv.page_table[(size_t)seq * kv.max_pages_per_seq + lp];
    if (page < 0) return nullptr;
    return reinterpret_cast<T*>(kv.base) + ((int64_t)page * kv.page_tokens + (pos & (kv.page_tokens - 1))) * kv.row;
}
// Row of (layer, which = 0 K / 1 V) holding position `pos` of stream `seq`; nullptr when the
// position is outside the reserved pages (the caller records TSB_DEV_BAD_INDEX and skips).
__device__ __forceinline__ __half* kv_row(const KvView& kv, int layer, int which, int seq, int pos) {
    const int lp = pos >> kv.page_shift;
    if (pos < 0 || lp >= kv.max_pages_per_seq) return nullptr;
    const int page = kv.page_table[(size_t)seq * kv.max_pages_per_seq + lp];
    if (page < 0) return nullptr;
    const int64_t row = (int64_t)kv.kv_heads * kv.head_dim;
    return kv.pool + (int64_t)layer * kv.layer_stride + (int64_t)which * kv.kv_stride +
           ((int64_t)page * kv.page_tokens + (pos & (kv.page_tokens - 1))) * row;
}
#endif
