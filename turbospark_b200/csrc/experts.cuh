// Routed feed-forwards of the plain-weight decoders: the choice of experts and the lists that the grouped products work from.
// Every (row, choice) pair of a pass gets a slot; the slots of an expert are consecutive, in row order.
#pragma once
#include "common.cuh"

struct ExpertChunk {
    int32_t expert, first, n;  // slots [first, first + n) of one expert
};
// Device buffers of a routed pass.
struct ExpertLists {
    int32_t* ids = nullptr;       // [rows, top]: chosen experts, best first
    float* weight = nullptr;      // [rows, top]
    int32_t* slot_of = nullptr;   // [rows, top]
    int32_t* token_of = nullptr;  // [slots]: the row a slot belongs to
    int32_t* first = nullptr;     // [experts + 1]: an expert's first slot
    ExpertChunk* chunks = nullptr;  // an expert's slots in runs of at most chunk_slots
    int32_t* n_chunks = nullptr;
};
// most chunks that `slots` pairs over n experts can make
inline int expert_chunks_max(int slots, int n, int chunk_slots) {
    const int64_t most = (int64_t)n + slots / chunk_slots;
    return (int)(most < slots ? most : slots);
}
constexpr int EXPERTS_MAX = 1024;

// Scores s = sigmoid(logits), choice = s + correction.  Of `groups` equal groups of neighbours the `keep` with the largest sum of their two
// largest choices stay; of their experts the `top` largest choices are taken (ties: the lower index), with weights s.
struct ExpertRouting {
    const float* logits = nullptr;  // [rows, logits_stride]
    int64_t logits_stride = 0;
    const float* correction = nullptr;
    int experts = 0, top = 0, groups = 1, keep = 1, rows = 0, chunk_slots = 16;
    ExpertLists lists{};
};
bool routing_supported(int experts, int top, int groups, int keep);
cudaError_t launch_route_experts(tsb_ctx* ctx, cudaStream_t st, const ExpertRouting& r);
// out[slot] = row token_of[slot] of x, `bytes` (a multiple of 16) per row
cudaError_t launch_gather_rows(tsb_ctx* ctx, cudaStream_t st, const void* x, int64_t x_bytes, const int32_t* token_of, int slots, void* out, int64_t bytes);
