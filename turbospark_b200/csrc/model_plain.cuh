// The plain-weight decoder family: tensors of a model and the work buffers of a session.
#pragma once
#include "attention_latent.cuh"
#include "attention_window.cuh"
#include "gemm_plain.cuh"
#include "model.cuh"
#include "recurrence.cuh"
#include "rowops_plain.cuh"
#include "scan.cuh"
#include "sublayer.cuh"

// attention: values that are the keys; values of their own; latent rows; none (the layer's mixer is a recurrence alone)
enum PlainMixer { MIX_KEYS = 0, MIX_KV = 1, MIX_LATENT = 2, MIX_NONE = 3 };

struct PlainLayer {
    tsb_plain_layer cfg{};
    PlainMixer mixer = MIX_KEYS;
    bool post_norm = false;    // one of the forms whose sublayers follow each other (post-norm, output norm, pre-norm)
    int tied = -1;             // the layer whose tensors this one uses
    int source = 0;            // the layer whose cache rows this one reads
    int head_pad = 0;          // head size the attention kernels work on; latent layers: columns of a head in q (and of an expanded key)
    int value_pad = 0;         // columns of a head in the attention's output
    int key_dim = 0, rank_pad = 0;  // latent layers: columns of a cached row, and of a head's sum of latents
    int q_rows = 0, k_rows = 0;
    int ffn_pad = 0;           // feed-forward width, padded
    int o_cols = 0;            // columns of the output projection before the feed-forward's (padded)
    int rotation = -1, value_rotation = -1;  // which of the model's rotations
    bool expands = false;      // long portions expand the latents to keys and values
    int rec_cols = 0;          // columns of the output projection that belong to the recurrence (padded), behind the heads'
    // parallel form: in = [queries | keys | head gates | (gate, up) pairs] x d, out = d x [heads | feed-forward]
    // post-norm form: in = [queries | keys | values] x d or [queries | latent | value gates | rotated pairs] x d, out = d x heads
    // output-norm form: in = [queries | keys | values | value gates | recurrence's vectors | recurrence's gates] x d, out = d x [heads | recurrence]
    PlainMat in, out;
    PlainMat ff_in, ff_out;    // forms whose sublayers follow each other; with experts: one expert's shape, the matrices one after another
    PlainMat router;
    float *in_bias = nullptr, *slopes = nullptr, *conv1 = nullptr, *conv2 = nullptr, *correction = nullptr;
    float *rec_lower = nullptr, *rec_norm = nullptr, *rec_conv = nullptr, *rec_conv_bias = nullptr, *rec_a_log = nullptr, *rec_skip = nullptr;
    // latent layers.  absorb: a head's query -> the latent's space (W_uk transposed, head by head); lift: a head's sum of latents ->
    // its values (W_uv); expand: latents -> every head's key and value
    PlainMat absorb, lift, expand;
    float *gain = nullptr, *mu = nullptr, *r1 = nullptr, *r2 = nullptr;
    float *norm2 = nullptr, *q_norm = nullptr, *k_norm = nullptr, *c_norm = nullptr, *sink = nullptr;
    uint64_t set = 0;          // bit per TSB_P_* uploaded
    bool owned = true;
    std::vector<void**> buffers() {
        return {&in.data, &out.data, &ff_in.data, &ff_out.data, &absorb.data, &lift.data, &expand.data, (void**)&gain, (void**)&mu, (void**)&r1, (void**)&r2,
                (void**)&norm2, (void**)&q_norm, (void**)&k_norm, (void**)&c_norm, (void**)&sink, &router.data, (void**)&in_bias, (void**)&slopes,
                (void**)&conv1, (void**)&conv2, (void**)&correction, (void**)&rec_lower, (void**)&rec_norm, (void**)&rec_conv, (void**)&rec_conv_bias,
                (void**)&rec_a_log, (void**)&rec_skip};
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
    void* positions = nullptr;  // [positions, d]
    float* final_gain = nullptr;  // [1], or [d] where the sublayers follow each other
    uint64_t set = 0;
    bool owned = true;
    bool any_shift = false;
    bool sequential() const { return cfg.post_norm || cfg.output_norm || cfg.pre_norm; }
    bool shifted_gains() const { return cfg.post_norm || cfg.pre_norm; }  // norm weights are given as their distance from one
};

// What the streams of an output-norm or pre-norm model keep from row to row.
struct StreamStates {
    int ring = 0;                           // states of a recurrence kept per stream
    int row_ring = 0, keep = 0;             // rows kept of a convolution's input; the most that any convolution looks back
    std::vector<RowRing> conv1, conv2, rec; // per layer: inputs of the two sublayers' convolutions and of the recurrence's
    std::vector<RecurrentState> states;     // per layer
    void* chunk_scratch = nullptr;          // of the chunked recurrences
    float2* scan_sums = nullptr;            // of the element-wise ones
    RowRing* rings_dev = nullptr;           // all rings that look back
    int n_rings = 0;
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
    // output-norm form; recurrences
    float *x2 = nullptr, *y = nullptr, *rec_out = nullptr, *router_logits = nullptr;
    void *rec = nullptr, *rec_mixed = nullptr, *expert_in = nullptr, *expert_act = nullptr, *expert_out = nullptr;
    int64_t rec_stride = 0, rec_mixed_stride = 0, rec_out_stride = 0, raw_rec = 0;  // raw_rec: where the recurrence's numbers start in a raw row
    int expert_rows = 0;   // slots the expert buffers hold
    ExpertLists lists;
    StreamStates states;
    void *gemm_ws = nullptr, *attn_ws = nullptr;
    ShiftState shift;
};
