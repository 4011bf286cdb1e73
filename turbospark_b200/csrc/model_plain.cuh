// The plain-weight decoder family: tensors of a model and the work buffers of a session.
#pragma once
#include "attention_latent.cuh"
#include "attention_window.cuh"
#include "gemm_plain.cuh"
#include "model.cuh"
#include "rowops_plain.cuh"

enum PlainMixer { MIX_KEYS = 0, MIX_KV = 1, MIX_LATENT = 2 };  // values that are the keys; values of their own; latent rows

struct PlainLayer {
    tsb_plain_layer cfg{};
    PlainMixer mixer = MIX_KEYS;
    bool post_norm = false;
    int source = 0;            // the layer whose cache rows this one reads
    int head_pad = 0;          // head size the attention kernels work on; latent layers: columns of a head in q (and of an expanded key)
    int value_pad = 0;         // columns of a head in the attention's output
    int key_dim = 0, rank_pad = 0;  // latent layers: columns of a cached row, and of a head's sum of latents
    int q_rows = 0, k_rows = 0;
    int ffn_pad = 0;           // feed-forward width, padded
    int o_cols = 0;            // columns of the output projection before the feed-forward's (padded)
    int rotation = -1;         // which of the model's rotations
    bool expands = false;      // long portions expand the latents to keys and values
    // parallel form: in = [queries | keys | head gates | (gate, up) pairs] x d, out = d x [heads | feed-forward]
    // post-norm form: in = [queries | keys | values] x d or [queries | latent | value gates | rotated pairs] x d, out = d x heads
    PlainMat in, out;
    PlainMat ff_in, ff_out;    // post-norm form
    // latent layers.  absorb: a head's query -> the latent's space (W_uk transposed, head by head); lift: a head's sum of latents ->
    // its values (W_uv); expand: latents -> every head's key and value
    PlainMat absorb, lift, expand;
    float *gain = nullptr, *mu = nullptr, *r1 = nullptr, *r2 = nullptr;
    float *norm2 = nullptr, *q_norm = nullptr, *k_norm = nullptr, *c_norm = nullptr, *sink = nullptr;
    uint32_t set = 0;          // bit per TSB_P_* uploaded
    bool owned = true;
    std::vector<void**> buffers() {
        return {&in.data, &out.data, &ff_in.data, &ff_out.data, &absorb.data, &lift.data, &expand.data, (void**)&gain, (void**)&mu, (void**)&r1, (void**)&r2,
                (void**)&norm2, (void**)&q_norm, (void**)&k_norm, (void**)&c_norm, (void**)&sink};
    }
};

// Frequencies of one kind of rotary position.
struct PlainRotation {
    int dims = 0;
    double base = 0, factor = 0, original = 0, fast = 0, slow = 0;
    double* freq = nullptr;    // device, [dims / 2]
    float magnitude = 1.f;
};

struct PlainModel {
    tsb_plain_config cfg{};
    bool f32 = false;
    int elem = 2;
    int64_t d_pad = 0;
    std::vector<PlainLayer> layers;
    std::vector<PlainRotation> rotations;
    PlainMat head;
    void* embed = nullptr;     // [vocab, d], natural rows
    float* final_gain = nullptr;  // [1], or [d] in a post-norm model
    uint32_t set = 0;
    bool owned = true;
    bool any_shift = false;
};

// Where the expansions of latents live: whole streams of a pass, in pages of EXPAND_PAGE positions.
constexpr int EXPAND_PAGE = 128;
struct ExpandRt {
    int pages = 0;             // 0: no expansion in this session
    int max_seqs = 0, pages_per_seq = 0;
    void *wide = nullptr, *latents = nullptr;
    int32_t* table = nullptr;  // [max_seqs][pages_per_seq]
};

struct PlainRt {
    int rows = 0;              // rows the buffers hold
    int64_t in_stride = 0, q_stride = 0, cat_stride = 0, act_stride = 0, raw_stride = 0, absorbed_stride = 0, sums_stride = 0, value_gate_stride = 0;
    int gate_stride = 0;
    float *x = nullptr, *gate = nullptr, *raw = nullptr;
    void *mix = nullptr, *h = nullptr, *q = nullptr, *cat = nullptr, *fin = nullptr;
    void *act = nullptr, *absorbed = nullptr, *sums = nullptr, *value_gate = nullptr;  // post-norm form
    std::vector<float2*> rotary;  // per rotation: [rows, dims / 2]
    ExpandRt expand;
    int fin_rows = 0;
    void *gemm_ws = nullptr, *attn_ws = nullptr;
    ShiftState shift;
};
