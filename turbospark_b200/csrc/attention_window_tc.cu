// The tcgen05 attention kernels for caches whose values are their keys.
#include "attention_window_tc.cuh"

bool wattn_tc_supported(int head_dim, int group, bool biased) {
    return (head_dim == 64 || head_dim == 128) && group >= 1 && group <= (biased ? WT_GROUP_MAX : WT_QM);
}

cudaError_t launch_window_attn_tc(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    return a.keys.head_dim == 64 ? launch_tc<64, 64, 128, false>(ctx, st, a, l, scratch) : launch_tc<128, 128, 128, false>(ctx, st, a, l, scratch);
}
