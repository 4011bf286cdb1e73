// The tcgen05 attention kernels for a window with a prefix before it.
#include "attention_window_tc.cuh"

cudaError_t launch_prefix_attn_tc(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    return a.keys.head_dim == 64 ? launch_tc<64, 64, 128, true, true>(ctx, st, a, l, scratch) : launch_tc<128, 128, 128, true, true>(ctx, st, a, l, scratch);
}
