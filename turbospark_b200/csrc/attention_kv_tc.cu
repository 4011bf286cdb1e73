// The tcgen05 attention kernels for caches with values of their own, and for keys and values of different widths.
#include "attention_window_tc.cuh"

cudaError_t launch_kv_attn_tc(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    return a.keys.head_dim == 64 ? launch_tc<64, 64, 128, true>(ctx, st, a, l, scratch) : launch_tc<128, 128, 128, true>(ctx, st, a, l, scratch);
}

bool wattn_wide_supported(int key_dim, int value_dim) {
    return (key_dim == 64 || key_dim == 128 || key_dim == 192) && (value_dim == 64 || value_dim == 128);
}

cudaError_t launch_window_attn_wide(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const AttnBatch& b, void* scratch) {
    WattnLaunch l{b.large, b.n_large, 1, 0, WATTN_WIDE_ROWS, b.max_len};
    if (b.rows_per_seq > 0) {
        const int tpg = (b.rows_per_seq + WATTN_WIDE_ROWS - 1) / WATTN_WIDE_ROWS;
        l = WattnLaunch{nullptr, b.rows / b.rows_per_seq * tpg, tpg, b.rows_per_seq, WATTN_WIDE_ROWS, b.max_len};
    }
    if (l.n_tiles == 0) return cudaSuccess;
    const int dk = a.keys.head_dim, dv = a.value_dim;
    if (dk == 64 && dv == 64) return launch_tc<64, 64, 128, true>(ctx, st, a, l, scratch);
    if (dk == 64 && dv == 128) return launch_tc<64, 128, 128, true>(ctx, st, a, l, scratch);
    if (dk == 128 && dv == 64) return launch_tc<128, 64, 128, true>(ctx, st, a, l, scratch);
    if (dk == 128 && dv == 128) return launch_tc<128, 128, 128, true>(ctx, st, a, l, scratch);
    if (dk == 192 && dv == 64) return launch_tc<192, 64, 64, true>(ctx, st, a, l, scratch);
    if (dk == 192 && dv == 128) return launch_tc<192, 128, 64, true>(ctx, st, a, l, scratch);
    return cudaErrorInvalidValue;
}
