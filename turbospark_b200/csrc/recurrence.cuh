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
    float* norm = nullptr;  // REC_MLSTM: [stream][ring][heads][dim]
    double* top = nullptr;  // REC_MLSTM: [stream][ring][heads]; in double, since the decay is the exponential of small differences of it
    int ring = 0, n_streams = 0;
};
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
};
constexpr int REC_MAX_DIM = 1024;

// Portions (whole portions of streams) row by row; the state after each of a portion's last `ring` rows is kept.
cudaError_t launch_recurrence_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const Recurrence& r, const RowTiles& portions);
// Long portions in bfloat16, REC_CHUNK rows at a time on the tensor cores; the state after the last row is kept.
constexpr int REC_CHUNK = 64;
bool recurrence_chunks_supported(int kind, int dim, int vdim);
cudaError_t launch_recurrence_chunks(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RowTiles& portions);
