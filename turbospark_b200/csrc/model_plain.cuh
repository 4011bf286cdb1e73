// The plain-weight decoder family: tensors of a model and the work buffers of a session.
#pragma once
#include "attention_window.cuh"
#include "gemm_plain.cuh"
#include "model.cuh"
#include "rowops_plain.cuh"

struct PlainLayer {
    tsb_plain_layer cfg{};
    int head_pad = 0;          // head size the kernels work on
    int q_rows = 0, k_rows = 0;
    int ffn_pad = 0;           // feed-forward width, padded
    int o_cols = 0;            // columns of the output projection before the feed-forward's (padded)
    PlainMat in, out;          // [queries | keys | head gates | (gate, up) pairs] x d;  d x [heads | feed-forward]
    float *gain = nullptr, *mu = nullptr, *r1 = nullptr, *r2 = nullptr;
    uint32_t set = 0;          // bit per TSB_P_* uploaded
    bool owned = true;
};

struct PlainModel {
    tsb_plain_config cfg{};
    bool f32 = false;
    int elem = 2;
    int64_t d_pad = 0;
    std::vector<PlainLayer> layers;
    PlainMat head;
    void* embed = nullptr;     // [vocab, d], natural rows
    float* final_gain = nullptr;
    uint32_t set = 0;
    bool owned = true;
    bool any_shift = false;
};

struct PlainRt {
    int rows = 0;              // rows the buffers hold
    int64_t in_stride = 0, q_stride = 0, cat_stride = 0;
    int gate_stride = 0;
    float *x = nullptr, *gate = nullptr;
    void *mix = nullptr, *h = nullptr, *q = nullptr, *cat = nullptr, *fin = nullptr;
    int fin_rows = 0;
    void *gemm_ws = nullptr, *attn_ws = nullptr;
    ShiftState shift;
};
