// Recurrent mixers: heads with a state S [dim, vdim] in f32,
//   S_t = decay_t S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t.
#pragma once
#include "stream_state.cuh"

enum RecurrenceKind {
    REC_FORGET = 1,  // q <- silu(q); decay per row of S: f = lower + (1 - lower) sigmoid(gate), k = 1 - f
    REC_MLSTM = 2,   // decay and input scale per head from two gates, stabilised by a running maximum; a normaliser n beside S
    REC_SSD = 3,     // decay exp(-exp(a_log) dt), k <- dt k, dt = softplus(gate); o <- o + skip * v
};

// States of one layer for every stream and the last `ring` positions (a power of two): position p in slot p & (ring - 1).
struct RecurrentState {
    float* s = nullptr;     // [stream][ring][heads][dim][v_pitch]
    // REC_MLSTM, a copy for every REC_COLS value columns (their owners read and write them at times of their own): [stream][ring][heads][copies][dim],
    // [stream][ring][heads][copies]
    float* norm = nullptr;
    double* top = nullptr;  // in double, since the decay is the exponential of small differences of it
    int ring = 0, n_streams = 0;
};
constexpr int REC_COLS = 32;
constexpr int recurrence_copies(int vdim) { return (vdim + REC_COLS - 1) / REC_COLS; }
constexpr int recurrence_v_pitch(int vdim) { return (vdim + 3) / 4 * 4; }

struct Recurrence {
    int kind = 0;
    int heads = 0, dim = 0, vdim = 0;
    int heads_per_key = 1;  // heads that share a q and a k
    const void *q = nullptr, *k = nullptr, *v = nullptr;  // the compute type; head h: q and k at (h / heads_per_key) * dim, v at h * vdim
    int64_t q_stride = 0, k_stride = 0, v_stride = 0;
    // pre-activations in f32: REC_FORGET [heads * dim] forget gates; REC_MLSTM [heads] input, then [heads] forget gates; REC_SSD [heads] steps
    const float* gate = nullptr;
    int64_t gate_stride = 0;
    const float* lower = nullptr;                    // REC_FORGET: [heads * dim]
    const float *a_log = nullptr, *skip = nullptr;   // REC_SSD: [heads]
    float cap = 0.f;                                 // REC_MLSTM
    float q_scale = 1.f;
    float* out = nullptr;                            // [rows, out_stride] f32, head h at h * vdim
    int64_t out_stride = 0;
    RecurrentState state{};
    const tsb_row_desc* rows = nullptr;
    int n_rows = 0;                                  // of the pass
};
constexpr int REC_MAX_DIM = 1024;

// Portions (whole portions of streams) row by row; the state after each of a portion's last `ring` rows is kept.
cudaError_t launch_recurrence_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const Recurrence& r, const RowTiles& portions);
// Long portions in bfloat16, REC_CHUNK rows at a time on the tensor cores; the state after a portion's last row is kept.  A portion's chunks
// are consecutive, in the list and in the scratch memory.
constexpr int REC_CHUNK = 64;
struct ChunkPortion {
    int32_t first_row, n_rows, first_chunk;
};
struct RecurrenceChunks {
    RowTiles chunks{};                       // all chunks of all portions, REC_CHUNK rows each but a portion's last
    const ChunkPortion* portions = nullptr;  // device; null: portions of rows_per_seq rows each
    int n_portions = 0, rows_per_seq = 0;
    void* scratch = nullptr;                 // recurrence_scratch_bytes for as many chunks
};
bool recurrence_chunks_supported(int kind, int dim, int vdim);
size_t recurrence_scratch_bytes(int kind, int heads, int dim, int vdim, int chunks);
cudaError_t launch_recurrence_chunks(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RecurrenceChunks& c);
