// Gated recurrences element by element (minGRU): S_t = (1 - z_t) S_(t-1) + z_t c_t per channel, out_t = S_t silu(g_t).
#pragma once
#include "recurrence.cuh"

// z = sigmoid of the first `width` numbers of a row of `gate`, c = p(u) of the next `width` with p(u) = u + 1/2 from zero on and sigmoid(u) below.
// States as in RecurrentState, one number per channel (its heads, dim and vdim are 1, 1, width): [stream][ring][pitch of width].
struct GatedScan {
    const float* gate = nullptr;      // [rows, gate_stride] f32
    int64_t gate_stride = 0;
    const void* out_gate = nullptr;   // g: [rows, out_gate_stride], the compute type
    int64_t out_gate_stride = 0;
    void* out = nullptr;              // [rows, out_stride], the compute type
    int64_t out_stride = 0;
    int width = 0;
    RecurrentState state{};
    const tsb_row_desc* rows = nullptr;
    int n_rows = 0;                   // of the pass
};
// Whole portions of streams, row by row; the state after each of a portion's last `ring` rows is kept.
cudaError_t launch_gated_scan_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const GatedScan& g, const RowTiles& portions);
// Long portions by chunks of SCAN_CHUNK rows (a portion's last one may be shorter), a portion's chunks one after another in the list.  several: some portion
// has more than one; sums: [chunks][width] then.
constexpr int SCAN_CHUNK = 128;
cudaError_t launch_gated_scan_chunks(tsb_ctx* ctx, cudaStream_t st, bool f32, const GatedScan& g, const RowTiles& chunks, bool several, float2* sums);
