// The mma.sync attention kernels for a window with a prefix before it: see attention_window.cu.
#include "attention_window_mma.cuh"

cudaError_t launch_prefix_attn_small(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int queries, void* scratch) {
    return launch_small<true, true>(ctx, st, a, l, queries, scratch);
}
cudaError_t launch_prefix_attn_large(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    return launch_large<8, 1, true, true>(ctx, st, a, l, scratch);
}
