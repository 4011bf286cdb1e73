// The block-quantised decoder family: models whose matrices are verbatim GGUF blocks (dense Llama-style layers,
// routed feed-forwards), their tensors, their work buffers inside a session, and their forward passes on the kernels
// of this library, with the reference's rounding points (f16 storage between operators, fp32 accumulation, bf16 norm
// weights).
//
// Op order of one layer (crates/runtime/src/families/llama/mod.rs:205-291,
// dense.rs:48-120), fused where two reference dispatches are adjacent:
//   [residual add +] RMSNorm -> qkv matmul (one matmul over q|k|v rows) ->
//   RoPE + K/V store -> split-KV attention -> o_proj matmul ->
//   residual add + RMSNorm -> gate|up matmul -> SiLU*up -> down matmul
// Every producer of a matmul input writes the matmul's activation operand
// directly, so a layer is 9 launches.
#include <algorithm>
#include <cstring>
#include <memory>
#include <new>
#include <vector>

#include "attention.cuh"
#include "model.cuh"

namespace {

__device__ __forceinline__ uint32_t mix32(uint32_t x) {
    x ^= x >> 16;
    x *= 0x7feb352du;
    x ^= x >> 15;
    x *= 0x846ca68bu;
    x ^= x >> 16;
    return x;
}

// Seeded synthetic blocks: every byte pseudo-random, then the scale fields are overwritten so the
// dequantised weights are finite, zero-mean and of standard deviation about 0.02.
__host__ __device__ inline int block_bytes_of(int qtype) {
    return qtype == TSB_Q4_K ? 144 : qtype == TSB_Q6_K ? 210 : qtype == TSB_Q5_K ? 176 : qtype == TSB_Q8_0 ? 34 : 17;
}

__global__ void fill_blocks_kernel(uint8_t* __restrict__ data, int64_t n_blocks, int qtype, uint32_t seed) {
    const int bb = block_bytes_of(qtype);
    for (int64_t b = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; b < n_blocks; b += (int64_t)gridDim.x * blockDim.x) {
        uint8_t* p = data + b * bb;
        uint32_t h = mix32((uint32_t)b * 0x9E3779B9u + seed) ^ mix32((uint32_t)(b >> 32) + seed * 31u);
        for (int i = 0; i < bb; i++) {
            if ((i & 3) == 0) h = mix32(h + 0x9E3779B9u);
            p[i] = (uint8_t)(h >> ((i & 3) * 8));
        }
        const float u = (float)(mix32(h) >> 8) * (1.0f / 16777216.0f);
        if (qtype == TSB_Q4_K) {
            // zero-mean weights of std ~0.02: E[sc*q] = 31.5*7.5 is cancelled by dmin*E[m] with dmin = 7.5 d
            const __half d = __float2half_rn(7.7e-5f * (0.5f + u)), dm = __float2half_rn(7.5f * 7.7e-5f * (0.5f + u));
            const unsigned short db = __half_as_ushort(d), mb = __half_as_ushort(dm);
            p[0] = db & 0xFF, p[1] = db >> 8, p[2] = mb & 0xFF, p[3] = mb >> 8;
        } else if (qtype == TSB_Q6_K) {
            const unsigned short db = __half_as_ushort(__float2half_rn(1.46e-5f * (0.5f + u)));
            p[208] = db & 0xFF, p[209] = db >> 8;
        } else if (qtype == TSB_Q5_K) {
            // E[sc*q] = 31.5*15.5 cancelled by dmin*E[m] with dmin = 15.5 d
            const __half d = __float2half_rn(3.7e-5f * (0.5f + u)), dm = __float2half_rn(15.5f * 3.7e-5f * (0.5f + u));
            const unsigned short db = __half_as_ushort(d), mb = __half_as_ushort(dm);
            p[0] = db & 0xFF, p[1] = db >> 8, p[2] = mb & 0xFF, p[3] = mb >> 8;
        } else if (qtype == TSB_Q8_0) {
            const unsigned short db = __half_as_ushort(__float2half_rn(2.7e-4f * (0.5f + u)));
            p[0] = db & 0xFF, p[1] = db >> 8;
        } else {
            p[0] = (uint8_t)(119 + (h & 1));
        }
    }
}

__global__ void fill_u16_kernel(uint16_t* p, int64_t n, uint16_t v) {
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) p[i] = v;
}

}  // namespace

// ------------------------------------------------------------------ model

static int64_t mat_bytes(const Mat& m) { return m.rows * tsb_row_bytes(m.qtype, m.cols); }

static int32_t mat_alloc(tsb_ctx* ctx, Mat& m, int qtype, int64_t rows, int64_t cols) {
    m.qtype = qtype, m.rows = rows, m.cols = cols;
    void* p = nullptr;
    // spare bytes: the bulk-copy path may over-fetch one 16-byte granule past an unaligned row run
    int32_t rc = tsb_alloc(ctx, (size_t)mat_bytes(m) + 256, &p);
    if (rc) return rc;
    m.data = (uint8_t*)p;
    m.owned = true;
    cudaMemset(m.data + mat_bytes(m), 0, 256);
    return TSB_OK;
}

static void mat_free(tsb_ctx* ctx, Mat& m) {
    if (m.owned && m.data) tsb_free(ctx, m.data);
    m = Mat();
}

static int local_experts(const tsb_model* m) { return m->n_local_experts > 0 ? m->n_local_experts : m->n_experts; }

static int64_t rows_of_v(const tsb_model_config& c) { return (int64_t)c.n_kv_heads * c.head_dim; }

extern const ModelFamily BLOCKS_FAMILY;

static Mat* fused_slot(tsb_model* m, int layer, int which, int64_t* row_off, int64_t* total_rows, int64_t* want_rows,
                       int64_t* want_cols) {
    const tsb_model_config& c = m->cfg;
    const int64_t qd = (int64_t)c.n_q_heads * c.head_dim, kd = (int64_t)c.n_kv_heads * c.head_dim;
    *row_off = 0;
    if (which == TSB_W_EMBED) {
        *total_rows = *want_rows = c.vocab, *want_cols = c.d_model;
        return &m->embed;
    }
    if (which == TSB_W_LM_HEAD) {
        *total_rows = *want_rows = c.vocab, *want_cols = c.d_model;
        return &m->lm_head;
    }
    if (layer < 0 || layer >= c.n_layers) return nullptr;
    LayerW& l = m->layers[layer];
    switch (which) {
        case TSB_W_Q: *total_rows = qd + 2 * kd, *want_rows = qd, *want_cols = c.d_model; return &l.wqkv;
        case TSB_W_K: *total_rows = qd + 2 * kd, *want_rows = kd, *want_cols = c.d_model, *row_off = qd; return &l.wqkv;
        case TSB_W_V: *total_rows = qd + 2 * kd, *want_rows = kd, *want_cols = c.d_model, *row_off = qd + kd; return &l.wqkv;
        case TSB_W_O: *total_rows = *want_rows = c.d_model, *want_cols = qd; return &l.wo;
        case TSB_W_GATE: *total_rows = 2 * (int64_t)c.ffn, *want_rows = c.ffn, *want_cols = c.d_model; return &l.wgu;
        case TSB_W_UP: *total_rows = 2 * (int64_t)c.ffn, *want_rows = c.ffn, *want_cols = c.d_model, *row_off = c.ffn; return &l.wgu;
        case TSB_W_DOWN: *total_rows = *want_rows = c.d_model, *want_cols = c.ffn; return &l.wdown;
        default: return nullptr;
    }
}

extern "C" {

int32_t tsb_model_create(tsb_ctx* ctx, const tsb_model_config* cfg, tsb_model** out) {
    if (!ctx || !cfg || !out) return TSB_ERR_INVALID;
    *out = nullptr;
    TSB_REQUIRE(ctx, cfg->n_layers > 0 && cfg->d_model > 0 && cfg->n_q_heads > 0 && cfg->n_kv_heads > 0 && cfg->ffn > 0 &&
                         cfg->vocab > 0 && cfg->max_context > 0,
                "model dimensions must be positive");
    TSB_REQUIRE(ctx, cfg->head_dim == 64 || cfg->head_dim == 128, "head_dim must be 64 or 128");
    TSB_REQUIRE(ctx, cfg->n_q_heads % cfg->n_kv_heads == 0, "n_q_heads must be a multiple of n_kv_heads");
    if (cfg->d_model % 256 || cfg->ffn % 256 || (cfg->n_q_heads * cfg->head_dim) % 256)
        return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "d_model, ffn and n_q_heads*head_dim must be multiples of 256");
    tsb_model* m = new (std::nothrow) tsb_model();
    if (!m) return TSB_ERR_OOM;
    m->ctx = ctx;
    m->family = &BLOCKS_FAMILY;
    m->cfg = *cfg;
    m->layers.resize(cfg->n_layers);
    *out = m;
    return TSB_OK;
}

int32_t tsb_model_set_matrix(tsb_model* m, int32_t layer, int32_t which, int32_t qtype, const void* host_blocks,
                             int64_t rows, int64_t cols) {
    if (!m) return TSB_ERR_INVALID;
    tsb_ctx* ctx = m->ctx;
    TSB_REQUIRE(ctx, m->family == &BLOCKS_FAMILY, "the model does not hold block-quantised tensors");
    TSB_REQUIRE(ctx, host_blocks, "null data");
    TSB_REQUIRE(ctx, qtype >= TSB_Q4_K && qtype <= TSB_QTYPE_LAST, "unknown block format %d", qtype);
    int64_t off, total, wr, wc;
    Mat* slot = fused_slot(m, layer, which, &off, &total, &wr, &wc);
    TSB_REQUIRE(ctx, slot, "no such tensor (layer %d, which %d)", layer, which);
    TSB_REQUIRE(ctx, rows == wr && cols == wc, "tensor %d of layer %d must be %lld x %lld, got %lld x %lld", which, layer,
                (long long)wr, (long long)wc, (long long)rows, (long long)cols);
    DeviceGuard g(ctx);
    const int64_t rb = tsb_row_bytes(qtype, cols);
    if (which == TSB_W_Q || which == TSB_W_K || which == TSB_W_V) {
        // Files quantized with mixed recipes keep v in a wider format than q and k: v then lives in its own matrix
        // and the pass runs the q|k rows and the v rows as two launches.
        LayerW& l = m->layers[layer];
        const int64_t qk_rows = total - rows_of_v(m->cfg);
        if (which == TSB_W_V && (l.wv.data || (l.wqkv.data && l.wqkv.qtype != qtype))) {
            if (l.wv.data && l.wv.qtype != qtype) mat_free(ctx, l.wv);
            if (!l.wv.data) {
                int32_t rc = mat_alloc(ctx, l.wv, qtype, rows, cols);
                if (rc) return rc;
            }
            if (l.wqkv.data) l.wqkv.rows = qk_rows;
            TSB_CUDA(ctx, cudaMemcpy(l.wv.data, host_blocks, (size_t)(rows * rb), cudaMemcpyHostToDevice));
            l.qkv_set |= 4;
            return TSB_OK;
        }
        if (which != TSB_W_V && l.wqkv.data && l.wqkv.qtype != qtype) {
            if (l.qkv_set != 4 || l.wv.data || !l.wqkv.owned)
                return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "q and k of a layer must share one block format");
            // only v has arrived so far: it moves to its own matrix and q|k start over in the new format
            const int64_t vb = tsb_row_bytes(l.wqkv.qtype, cols);
            int32_t rc = mat_alloc(ctx, l.wv, l.wqkv.qtype, rows_of_v(m->cfg), cols);
            if (rc) return rc;
            TSB_CUDA(ctx, cudaMemcpy(l.wv.data, l.wqkv.data + qk_rows * vb, (size_t)(rows_of_v(m->cfg) * vb), cudaMemcpyDeviceToDevice));
            mat_free(ctx, l.wqkv);
            if ((rc = mat_alloc(ctx, l.wqkv, qtype, qk_rows, cols))) return rc;
        }
        l.qkv_set |= which == TSB_W_Q ? 1 : (which == TSB_W_K ? 2 : 4);
    }
    if (!slot->data) {
        int32_t rc = mat_alloc(ctx, *slot, qtype, total, cols);
        if (rc) return rc;
    } else if (slot->qtype != qtype) {
        return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "gate and up of a layer must share one block format");
    }
    TSB_CUDA(ctx, cudaMemcpy(slot->data + off * rb, host_blocks, (size_t)(rows * rb), cudaMemcpyHostToDevice));
    return TSB_OK;
}

int32_t tsb_model_set_moe(tsb_model* m, int32_t n_experts, int32_t top_k, int32_t moe_ffn) {
    if (!m) return TSB_ERR_INVALID;
    tsb_ctx* ctx = m->ctx;
    TSB_REQUIRE(ctx, m->family == &BLOCKS_FAMILY, "the model does not hold block-quantised tensors");
    TSB_REQUIRE(ctx, n_experts >= 1 && n_experts <= 512 && top_k >= 1 && top_k <= 8 && top_k <= n_experts, "need 1 <= top_k <= min(8, experts) and at most 512 experts");
    TSB_REQUIRE(ctx, moe_ffn > 0 && moe_ffn % 256 == 0, "the expert width must be a multiple of 256");
    for (const LayerW& l : m->layers) TSB_REQUIRE(ctx, !l.wgu.data && !l.wdown.data, "set_moe comes before the tensors");
    m->n_experts = n_experts, m->top_k = top_k, m->moe_ffn = moe_ffn;
    m->expert_lo = 0, m->n_local_experts = 0;
    return TSB_OK;
}

int32_t tsb_model_set_expert_shard(tsb_model* m, int32_t expert_lo, int32_t n_local) {
    if (!m) return TSB_ERR_INVALID;
    tsb_ctx* ctx = m->ctx;
    TSB_REQUIRE(ctx, m->family == &BLOCKS_FAMILY, "the model does not hold block-quantised tensors");
    TSB_REQUIRE(ctx, m->n_experts > 0, "the model has no experts (tsb_model_set_moe first)");
    TSB_REQUIRE(ctx, expert_lo >= 0 && n_local >= 1 && expert_lo + n_local <= m->n_experts, "experts %d..%d outside the model's %d", expert_lo,
                expert_lo + n_local, m->n_experts);
    for (const LayerW& l : m->layers) TSB_REQUIRE(ctx, !l.experts_gate_up && !l.experts_down, "the shard comes before the expert tensors");
    m->expert_lo = expert_lo, m->n_local_experts = n_local;
    return TSB_OK;
}

static int32_t upload(tsb_ctx* ctx, void** slot, const void* host, size_t bytes) {
    if (!*slot) {
        // spare bytes for the bulk-copy path's 16-byte granules, as for the dense matrices
        int32_t rc = tsb_alloc(ctx, bytes + 256, slot);
        if (rc) return rc;
        cudaMemset((uint8_t*)*slot + bytes, 0, 256);
    }
    TSB_CUDA(ctx, cudaMemcpy(*slot, host, bytes, cudaMemcpyHostToDevice));
    return TSB_OK;
}

int32_t tsb_model_set_router(tsb_model* m, int32_t layer, const void* q_u8, const void* scale_bf16, const void* bias_bf16) {
    if (!m) return TSB_ERR_INVALID;
    tsb_ctx* ctx = m->ctx;
    TSB_REQUIRE(ctx, m->family == &BLOCKS_FAMILY, "the model does not hold block-quantised tensors");
    TSB_REQUIRE(ctx, m->n_experts > 0, "the model has no experts (tsb_model_set_moe first)");
    TSB_REQUIRE(ctx, layer >= 0 && layer < m->cfg.n_layers && q_u8 && scale_bf16 && bias_bf16, "bad layer or null data");
    TSB_REQUIRE(ctx, m->cfg.d_model % 64 == 0, "d_model must be a multiple of the router's 64-column group");
    DeviceGuard g(ctx);
    LayerW& l = m->layers[layer];
    l.moe_owned = true;
    const size_t n = (size_t)m->n_experts * m->cfg.d_model;
    int32_t rc;
    if ((rc = upload(ctx, (void**)&l.router_q, q_u8, n)) || (rc = upload(ctx, (void**)&l.router_scale, scale_bf16, n / 64 * 2)) ||
        (rc = upload(ctx, (void**)&l.router_bias, bias_bf16, n / 64 * 2)))
        return rc;
    return TSB_OK;
}

int32_t tsb_model_set_experts(tsb_model* m, int32_t layer, int32_t qtype, const void* gate_up_blocks, const void* down_blocks) {
    if (!m) return TSB_ERR_INVALID;
    tsb_ctx* ctx = m->ctx;
    TSB_REQUIRE(ctx, m->family == &BLOCKS_FAMILY, "the model does not hold block-quantised tensors");
    TSB_REQUIRE(ctx, m->n_experts > 0, "the model has no experts (tsb_model_set_moe first)");
    TSB_REQUIRE(ctx, layer >= 0 && layer < m->cfg.n_layers && gate_up_blocks && down_blocks, "bad layer or null data");
    TSB_REQUIRE(ctx, qtype >= TSB_Q4_K && qtype <= TSB_QTYPE_LAST, "unknown block format %d", qtype);
    DeviceGuard g(ctx);
    LayerW& l = m->layers[layer];
    l.moe_owned = true;
    l.experts_qtype = qtype;
    const size_t gu = (size_t)local_experts(m) * 2 * m->moe_ffn * tsb_row_bytes(qtype, m->cfg.d_model);
    const size_t dn = (size_t)local_experts(m) * m->cfg.d_model * tsb_row_bytes(qtype, m->moe_ffn);
    int32_t rc;
    if ((rc = upload(ctx, (void**)&l.experts_gate_up, gate_up_blocks, gu)) || (rc = upload(ctx, (void**)&l.experts_down, down_blocks, dn))) return rc;
    return TSB_OK;
}

int32_t tsb_model_set_norm(tsb_model* m, int32_t layer, int32_t which, const void* host_bf16, int32_t n) {
    if (!m) return TSB_ERR_INVALID;
    tsb_ctx* ctx = m->ctx;
    TSB_REQUIRE(ctx, m->family == &BLOCKS_FAMILY, "the model does not hold block-quantised tensors");
    TSB_REQUIRE(ctx, host_bf16 && n == m->cfg.d_model, "a norm weight has d_model entries");
    uint16_t** slot;
    if (which == TSB_N_OUT) {
        slot = &m->out_norm;
        m->out_norm_owned = true;
    } else {
        TSB_REQUIRE(ctx, layer >= 0 && layer < m->cfg.n_layers, "layer %d outside the model", layer);
        slot = which == TSB_N_ATTN ? &m->layers[layer].attn_norm : &m->layers[layer].ffn_norm;
        m->layers[layer].norms_owned = true;
    }
    DeviceGuard g(ctx);
    if (!*slot) {
        void* p;
        int32_t rc = tsb_alloc(ctx, (size_t)n * 2, &p);
        if (rc) return rc;
        *slot = (uint16_t*)p;
    }
    TSB_CUDA(ctx, cudaMemcpy(*slot, host_bf16, (size_t)n * 2, cudaMemcpyHostToDevice));
    return TSB_OK;
}

int32_t tsb_model_fill_synthetic(tsb_model* m, int32_t qtype, int32_t lm_head_qtype, uint64_t seed) {
    if (!m) return TSB_ERR_INVALID;
    tsb_ctx* ctx = m->ctx;
    TSB_REQUIRE(ctx, m->family == &BLOCKS_FAMILY, "the model does not hold block-quantised tensors");
    TSB_REQUIRE(ctx, qtype >= TSB_Q4_K && qtype <= TSB_QTYPE_LAST && lm_head_qtype >= TSB_Q4_K && lm_head_qtype <= TSB_QTYPE_LAST, "bad format");
    DeviceGuard g(ctx);
    const tsb_model_config& c = m->cfg;
    const int64_t qd = (int64_t)c.n_q_heads * c.head_dim, kd = (int64_t)c.n_kv_heads * c.head_dim;
    uint32_t sd = (uint32_t)seed * 2654435761u + (uint32_t)(seed >> 32);
    auto fill = [&](Mat& t, int qt, int64_t rows, int64_t cols) -> int32_t {
        if (!t.data) {
            int32_t rc = mat_alloc(ctx, t, qt, rows, cols);
            if (rc) return rc;
        }
        const int64_t nb = mat_bytes(t) / block_bytes_of(qt);
        fill_blocks_kernel<<<1024, 256>>>(t.data, nb, qt, sd);
        sd = sd * 1664525u + 1013904223u;
        return TSB_OK;
    };
    auto ones = [&](uint16_t** p) -> int32_t {
        if (!*p) {
            void* q;
            int32_t rc = tsb_alloc(ctx, (size_t)c.d_model * 2, &q);
            if (rc) return rc;
            *p = (uint16_t*)q;
        }
        fill_u16_kernel<<<32, 256>>>(*p, c.d_model, (uint16_t)0x3F80);  // bf16 1.0
        return TSB_OK;
    };
    int32_t rc;
    for (auto& l : m->layers) {
        if ((rc = fill(l.wqkv, qtype, qd + 2 * kd, c.d_model))) return rc;
        if ((rc = fill(l.wo, qtype, c.d_model, qd))) return rc;
        if (m->n_experts > 0) {
            // routed layers: random 8-bit router with scale 0.004 / bias -0.5 (zero-mean weights), experts as blocks
            const size_t rn = (size_t)m->n_experts * c.d_model, rg = rn / 64;
            const int64_t gu_b = (int64_t)local_experts(m) * 2 * m->moe_ffn * tsb_row_bytes(qtype, c.d_model);
            const int64_t dn_b = (int64_t)local_experts(m) * c.d_model * tsb_row_bytes(qtype, m->moe_ffn);
            l.moe_owned = true, l.experts_qtype = qtype;
            void* p;
            if (!l.router_q) {
                if ((rc = tsb_alloc(ctx, rn + 256, &p))) return rc;
                l.router_q = (uint8_t*)p;
                if ((rc = tsb_alloc(ctx, rg * 2, &p))) return rc;
                l.router_scale = (uint16_t*)p;
                if ((rc = tsb_alloc(ctx, rg * 2, &p))) return rc;
                l.router_bias = (uint16_t*)p;
                if ((rc = tsb_alloc(ctx, (size_t)gu_b + 256, &p))) return rc;
                l.experts_gate_up = (uint8_t*)p;
                if ((rc = tsb_alloc(ctx, (size_t)dn_b + 256, &p))) return rc;
                l.experts_down = (uint8_t*)p;
                cudaMemset(l.experts_gate_up + gu_b, 0, 256), cudaMemset(l.experts_down + dn_b, 0, 256);
            }
            fill_blocks_kernel<<<64, 256>>>(l.router_q, (int64_t)(rn / 17), TSB_MXFP4, sd);  // any bytes do for the 8-bit weights
            fill_u16_kernel<<<32, 256>>>(l.router_scale, (int64_t)rg, (uint16_t)0x3B83);      // bf16 0.004
            fill_u16_kernel<<<32, 256>>>(l.router_bias, (int64_t)rg, (uint16_t)0xBF00);       // bf16 -0.5
            fill_blocks_kernel<<<1024, 256>>>(l.experts_gate_up, gu_b / block_bytes_of(qtype), qtype, sd + 1);
            fill_blocks_kernel<<<1024, 256>>>(l.experts_down, dn_b / block_bytes_of(qtype), qtype, sd + 2);
            sd = sd * 1664525u + 1013904223u;
        } else {
            if ((rc = fill(l.wgu, qtype, 2 * (int64_t)c.ffn, c.d_model))) return rc;
            if ((rc = fill(l.wdown, qtype, c.d_model, c.ffn))) return rc;
        }
        l.norms_owned = true;
        if ((rc = ones(&l.attn_norm)) || (rc = ones(&l.ffn_norm))) return rc;
    }
    if ((rc = fill(m->embed, qtype, c.vocab, c.d_model))) return rc;
    if ((rc = fill(m->lm_head, lm_head_qtype, c.vocab, c.d_model))) return rc;
    m->out_norm_owned = true;
    if ((rc = ones(&m->out_norm))) return rc;
    TSB_CUDA(ctx, cudaDeviceSynchronize());
    return TSB_OK;
}

}  // extern "C"

static void blocks_free_tensors(tsb_model* m) {
    for (auto& l : m->layers) {
        mat_free(m->ctx, l.wqkv), mat_free(m->ctx, l.wv), mat_free(m->ctx, l.wo), mat_free(m->ctx, l.wgu), mat_free(m->ctx, l.wdown);
        if (l.norms_owned) {
            if (l.attn_norm) tsb_free(m->ctx, l.attn_norm);
            if (l.ffn_norm) tsb_free(m->ctx, l.ffn_norm);
        }
        if (l.moe_owned)
            for (void* p : {(void*)l.router_q, (void*)l.router_scale, (void*)l.router_bias, (void*)l.experts_gate_up, (void*)l.experts_down})
                if (p) tsb_free(m->ctx, p);
    }
    mat_free(m->ctx, m->embed), mat_free(m->ctx, m->lm_head);
    if (m->out_norm_owned && m->out_norm) tsb_free(m->ctx, m->out_norm);
}

static int32_t blocks_share(tsb_model* dst, int32_t dst_layer, const tsb_model* src, int32_t src_layer) {
    tsb_ctx* ctx = dst->ctx;
    TSB_REQUIRE(ctx, dst->cfg.d_model == src->cfg.d_model && dst->cfg.vocab == src->cfg.vocab, "models differ in width or vocabulary");
    auto borrow = [](Mat& d, const Mat& s) {
        d = s;
        d.owned = false;
    };
    if (dst_layer < 0) {
        borrow(dst->embed, src->embed), borrow(dst->lm_head, src->lm_head);
        dst->out_norm = src->out_norm, dst->out_norm_owned = false;
        return TSB_OK;
    }
    TSB_REQUIRE(ctx, dst_layer < dst->cfg.n_layers && src_layer >= 0 && src_layer < src->cfg.n_layers, "layer out of range");
    TSB_REQUIRE(ctx, dst->cfg.ffn == src->cfg.ffn && dst->cfg.n_q_heads == src->cfg.n_q_heads &&
                         dst->cfg.n_kv_heads == src->cfg.n_kv_heads && dst->cfg.head_dim == src->cfg.head_dim,
                "layer shapes differ");
    LayerW& d = dst->layers[dst_layer];
    const LayerW& s = src->layers[src_layer];
    borrow(d.wqkv, s.wqkv), borrow(d.wv, s.wv), borrow(d.wo, s.wo), borrow(d.wgu, s.wgu), borrow(d.wdown, s.wdown);
    d.qkv_set = s.qkv_set;
    d.router_q = s.router_q, d.router_scale = s.router_scale, d.router_bias = s.router_bias;
    d.experts_gate_up = s.experts_gate_up, d.experts_down = s.experts_down, d.experts_qtype = s.experts_qtype, d.moe_owned = false;
    d.attn_norm = s.attn_norm, d.ffn_norm = s.ffn_norm, d.norms_owned = false;
    return TSB_OK;
}

static int64_t blocks_weight_bytes(const tsb_model* m) {
    int64_t t = mat_bytes(m->lm_head);
    for (auto& l : m->layers) t += mat_bytes(l.wqkv) + mat_bytes(l.wv) + mat_bytes(l.wo) + mat_bytes(l.wgu) + mat_bytes(l.wdown);
    if (m->n_experts > 0)  // every expert, although a pass reads only the routed ones
        for (auto& l : m->layers)
            t += (int64_t)local_experts(m) * (2 * m->moe_ffn * tsb_row_bytes(l.experts_qtype, m->cfg.d_model) +
                                          m->cfg.d_model * tsb_row_bytes(l.experts_qtype, m->moe_ffn)) +
                 (int64_t)m->n_experts * m->cfg.d_model;
    return t;
}

constexpr int WIDE_MIN_ROWS = 24;  // a model whose largest pass has this many rows or more runs every pass on the tensor-memory matmul

static int32_t blocks_complete(const tsb_model* m) {
    tsb_ctx* ctx = m->ctx;
    for (size_t i = 0; i < m->layers.size(); i++) {
        const LayerW& l = m->layers[i];
        if (m->n_experts > 0)
            TSB_REQUIRE(ctx, l.wqkv.data && l.wo.data && l.attn_norm && l.ffn_norm && l.router_q && l.experts_gate_up && l.experts_down,
                        "layer %zu is missing a tensor (attention, norms, router or experts)", i);
        else
            TSB_REQUIRE(ctx, l.wqkv.data && l.wo.data && l.wgu.data && l.wdown.data && l.attn_norm && l.ffn_norm,
                        "layer %zu is missing a tensor", i);
        TSB_REQUIRE(ctx, l.qkv_set == 0 || l.qkv_set == 7, "layer %zu is missing one of q, k, v", i);
    }
    TSB_REQUIRE(ctx, m->embed.data && m->lm_head.data && m->out_norm, "embedding, head or final norm missing");
    return TSB_OK;
}

static int32_t blocks_runtime_init(tsb_session* s, ModelRt& rt, const tsb_model* model, const SessionShape& shape, bool is_draft) {
    tsb_ctx* ctx = s->ctx;
    rt.model = model;
    const tsb_model_config& c = model->cfg;
    const int n_streams = shape.n_streams, max_rows = shape.max_rows;
    const int R = n_streams * max_rows;
    const int Rp = (R + 7) / 8 * 8;  // activation operands hold whole token tiles
    const int64_t qkv_dim = (int64_t)(c.n_q_heads + 2 * c.n_kv_heads) * c.head_dim;
    int32_t rc = tsb_kv_create(ctx, c.n_layers, c.n_kv_heads, c.head_dim, shape.page_tokens, shape.num_pages, n_streams,
                               shape.pages_per_seq, &rt.kv);
    if (rc) return rc;
    auto A = [&](size_t bytes, void** p) { return dev_alloc(ctx, s->owned, bytes, p); };
    if ((rc = A((size_t)R * c.d_model * 2, (void**)&rt.h))) return rc;
    if ((rc = A((size_t)R * c.n_q_heads * c.head_dim * 2, (void**)&rt.q))) return rc;
    if ((rc = A((size_t)R * c.head_dim * sizeof(float), (void**)&rt.cs))) return rc;
    if ((rc = A((size_t)(2 * c.n_layers + 1) * R * (c.d_model / 16) * sizeof(float), (void**)&rt.ss))) return rc;
    const int64_t od = (int64_t)c.n_q_heads * c.head_dim;
    if ((rc = A(act_xp_bytes(Rp, c.d_model), (void**)&rt.act_d.xp)) || (rc = A(act_xs_bytes(Rp, c.d_model), (void**)&rt.act_d.xs))) return rc;
    if ((rc = A(act_xp_bytes(Rp, od), (void**)&rt.act_o.xp)) || (rc = A(act_xs_bytes(Rp, od), (void**)&rt.act_o.xs))) return rc;
    if ((rc = A(act_xp_bytes(Rp, c.ffn), (void**)&rt.act_f.xp)) || (rc = A(act_xs_bytes(Rp, c.ffn), (void**)&rt.act_f.xs))) return rc;
    cudaMemset(rt.act_d.xp, 0, act_xp_bytes(Rp, c.d_model));
    cudaMemset(rt.act_o.xp, 0, act_xp_bytes(Rp, od));
    cudaMemset(rt.act_f.xp, 0, act_xp_bytes(Rp, c.ffn));
    cudaMemset(rt.act_d.xs, 0, act_xs_bytes(Rp, c.d_model));
    cudaMemset(rt.act_o.xs, 0, act_xs_bytes(Rp, od));
    cudaMemset(rt.act_f.xs, 0, act_xs_bytes(Rp, c.ffn));
    rt.attn_scratch_bytes = attn_scratch_bytes(R, c.n_q_heads, c.head_dim);
    if ((rc = A(rt.attn_scratch_bytes, &rt.attn_scratch))) return rc;
    cudaMemset(rt.attn_scratch, 0, rt.attn_scratch_bytes);  // the ticket words start at zero
    rt.fed.assign(n_streams, std::vector<int32_t>());
    rt.pending.assign(n_streams, PendingVerify());
    // the many-row path: only when the session can hold that many rows and every matrix suits the kernel
    if (model->n_experts > 0) {
        // routed feed-forward: natural-layout rows around the router and the experts
        if ((rc = A((size_t)R * c.d_model * 2, (void**)&rt.w_xn)) || (rc = A((size_t)R * qkv_dim * 2, (void**)&rt.w_qkv)) ||
            (rc = A((size_t)R * c.d_model * 2, (void**)&rt.w_o)) || (rc = A((size_t)R * model->n_experts * sizeof(float), (void**)&rt.moe_logits)) ||
            (rc = A((size_t)R * model->top_k * sizeof(int32_t), (void**)&rt.moe_ids)) || (rc = A((size_t)R * model->top_k * 2, (void**)&rt.moe_w)) ||
            (rc = A((size_t)R * c.d_model * 2, (void**)&rt.moe_zero)) ||
            (rc = A(moe_ffn_workspace_bytes(R, model->top_k, model->n_experts, c.d_model, model->moe_ffn), &rt.moe_ws)))
            return rc;
        cudaMemset(rt.moe_zero, 0, (size_t)R * c.d_model * 2);
        if ((rc = A((size_t)R * sizeof(float), (void**)&rt.moe_unit_ss))) return rc;
        if ((rc = A((size_t)R * c.d_model * sizeof(float), (void**)&rt.tp_partial))) return rc;
        {
            std::vector<float> unit((size_t)R, (float)c.d_model);  // sum / d_model = 1 and eps = 0: 1/rms = 1 exactly
            TSB_CUDA(ctx, cudaMemcpy(rt.moe_unit_ss, unit.data(), unit.size() * sizeof(float), cudaMemcpyHostToDevice));
        }
        return TSB_OK;
    }
    // One matmul path per (session, model), whatever a pass's row count: the register path and the tensor-memory path
    // sum in different orders, so a model that switched between them by row count would not reproduce its own
    // single-row results in a batch (the reference's verify runs the decode path's arithmetic).  The tensor-memory path
    // is taken when the model's largest pass has WIDE_MIN_ROWS rows or more: the target's verify carries max_rows rows
    // of every stream; the drafter's largest pass is two rows per stream (a round's first step) or one stream's tree.
    const int largest_pass = is_draft ? std::max(2 * n_streams, max_rows) : R;
    bool wide = largest_pass >= WIDE_MIN_ROWS && gemm_wide_supported(model->lm_head.qtype, model->lm_head.rows, model->lm_head.cols, R);
    for (const LayerW& l : model->layers)
        wide = wide && !l.wv.data && gemm_wide_supported(l.wqkv.qtype, l.wqkv.rows, l.wqkv.cols, R) && gemm_wide_supported(l.wo.qtype, l.wo.rows, l.wo.cols, R) &&
               gemm_wide_supported(l.wgu.qtype, l.wgu.rows, l.wgu.cols, R) && gemm_wide_supported(l.wdown.qtype, l.wdown.rows, l.wdown.cols, R);
    {
        const char* env = getenv("TSB_WIDE_FORWARD");
        if (env && env[0] == '0') wide = false;
    }
    if (wide) {
        const int64_t widest = std::max<int64_t>(std::max<int64_t>(c.d_model, od), c.ffn);
        if ((rc = A((size_t)R * c.d_model * 2, (void**)&rt.w_xn)) || (rc = A((size_t)R * qkv_dim * 2, (void**)&rt.w_qkv)) ||
            (rc = A((size_t)R * od * 2, (void**)&rt.w_ao)) || (rc = A((size_t)R * c.d_model * 2, (void**)&rt.w_o)) ||
            (rc = A((size_t)R * 2 * c.ffn * 2, (void**)&rt.w_gu)) || (rc = A((size_t)R * c.ffn * 2, (void**)&rt.w_a)) ||
            (rc = A((size_t)R * c.vocab * 2, (void**)&rt.w_logits)) || (rc = A(gemm_wide_workspace_bytes(widest, R), &rt.w_ws)))
            return rc;
        size_t part = gemm_wide_partial_bytes(ctx, model->lm_head.rows, model->lm_head.cols);
        for (const LayerW& l : model->layers)
            for (const Mat* mt : {&l.wqkv, &l.wo, &l.wgu, &l.wdown}) part = std::max(part, gemm_wide_partial_bytes(ctx, mt->rows, mt->cols));
        if (part && (rc = A(part, &rt.w_part))) return rc;
        if (part) TSB_CUDA(ctx, cudaMemset(rt.w_part, 0, 4096));  // the ticket words of cut tiles
        rt.wide_ok = true;
    }
    return TSB_OK;
}

// The same pass for many rows: natural-layout f16 activations, the tensor-memory matmul, and the reference's own
// operator order and rounding points (rms_norm -> matmul -> rope/store -> attention -> o_proj -> residual + rms_norm ->
// gate|up -> silu*up -> down -> residual; crates/runtime/src/families/llama/mod.rs:205-291).
static cudaError_t forward_device_wide(tsb_session* s, ModelRt& rt, const int32_t* tokens_dev, int token_stride,
                                       const tsb_row_desc* rows_dev, int rows, int rows_per_seq, int max_len, __half* logits,
                                       int64_t logits_stride, bool last_rows_only) {
    tsb_ctx* ctx = s->ctx;
    cudaStream_t st = s->stream;
    const tsb_model* m = rt.model;
    const tsb_model_config& c = m->cfg;
    const float scale = 1.0f / sqrtf((float)c.head_dim);
    const int64_t od = (int64_t)c.n_q_heads * c.head_dim, qkv_dim = (int64_t)(c.n_q_heads + 2 * c.n_kv_heads) * c.head_dim;
    const ActOut none{nullptr, nullptr};
    cudaError_t e;
#define FW(x)                           \
    do {                                \
        e = (x);                        \
        if (e != cudaSuccess) return e; \
    } while (0)
    FW(launch_embed_rows(ctx, st, m->embed.qtype, m->embed.data, c.vocab, c.d_model, tokens_dev, token_stride, rows, rt.h, 1.0f));
    FW(launch_rmsnorm_rows(ctx, st, rt.h, nullptr, m->layers[0].attn_norm, rt.w_xn, none, rows, c.d_model, c.rms_eps));
    for (int L = 0; L < c.n_layers; L++) {
        const LayerW& l = m->layers[L];
        FW(launch_gemm_wide_q4k(ctx, st, l.wqkv.data, l.wqkv.rows, l.wqkv.cols, rt.w_xn, c.d_model, rows, rt.w_qkv, qkv_dim, false, rt.w_ws, rt.w_part));
        FW(launch_rope_store_kv(ctx, st, rt.kv, L, rt.w_qkv, rows_dev, rows, c.n_q_heads, c.rope_theta));
        FW(launch_attn_decode_rows(ctx, st, rt.kv, L, rt.w_qkv, qkv_dim, rt.w_ao, none, rows_dev, rows, rows_per_seq, c.n_q_heads, scale,
                                   max_len, rt.attn_scratch, s->n_streams * s->max_rows));
        FW(launch_gemm_wide_q4k(ctx, st, l.wo.data, l.wo.rows, l.wo.cols, rt.w_ao, od, rows, rt.w_o, c.d_model, false, rt.w_ws, rt.w_part));
        FW(launch_rmsnorm_rows(ctx, st, rt.h, rt.w_o, l.ffn_norm, rt.w_xn, none, rows, c.d_model, c.rms_eps));
        FW(launch_gemm_wide_q4k(ctx, st, l.wgu.data, l.wgu.rows, l.wgu.cols, rt.w_xn, c.d_model, rows, rt.w_gu, 2 * (int64_t)c.ffn, false, rt.w_ws, rt.w_part));
        FW(launch_silu_mul(ctx, st, rt.w_gu, rt.w_gu + c.ffn, rt.w_a, none, rows, c.ffn, 2 * (int64_t)c.ffn, c.ffn));
        FW(launch_gemm_wide_q4k(ctx, st, l.wdown.data, l.wdown.rows, l.wdown.cols, rt.w_a, c.ffn, rows, rt.w_o, c.d_model, false, rt.w_ws, rt.w_part));
        const void* g = L + 1 < c.n_layers ? (const void*)m->layers[L + 1].attn_norm : (const void*)m->out_norm;
        FW(launch_rmsnorm_rows(ctx, st, rt.h, rt.w_o, g, rt.w_xn, none, rows, c.d_model, c.rms_eps));
    }
    if (logits) {
        if (last_rows_only && rows_per_seq > 1) {
            // every row's logits into the staging buffer, then each stream's last row to its place
            FW(launch_gemm_wide_q4k(ctx, st, m->lm_head.data, m->lm_head.rows, m->lm_head.cols, rt.w_xn, c.d_model, rows, rt.w_logits, c.vocab,
                                    false, rt.w_ws, rt.w_part));
            FW(cudaMemcpy2DAsync(logits, (size_t)logits_stride * 2, rt.w_logits + (size_t)(rows_per_seq - 1) * c.vocab,
                                 (size_t)rows_per_seq * c.vocab * 2, (size_t)c.vocab * 2, (size_t)(rows / rows_per_seq),
                                 cudaMemcpyDeviceToDevice, st));
        } else {
            FW(launch_gemm_wide_q4k(ctx, st, m->lm_head.data, m->lm_head.rows, m->lm_head.cols, rt.w_xn, c.d_model, rows, logits, logits_stride,
                                    false, rt.w_ws, rt.w_part));
        }
    }
#undef FW
    return cudaSuccess;
}

// The pass of a model whose feed-forward is routed (crates/runtime/src/families/llama/mod.rs:205-291 with the
// feed-forward of families/llama/moe.rs:36-221): unfused operators on natural-layout f16 rows with the reference's
// rounding points; the routed sum is formed over a zero residual and added to the stream afterwards.
static cudaError_t forward_device_moe(tsb_session* s, ModelRt& rt, const int32_t* tokens_dev, int token_stride,
                                      const tsb_row_desc* rows_dev, int rows, int rows_per_seq, int max_len, __half* logits,
                                      int64_t logits_stride, bool last_rows_only) {
    tsb_ctx* ctx = s->ctx;
    cudaStream_t st = s->stream;
    const tsb_model* m = rt.model;
    const tsb_model_config& c = m->cfg;
    const float scale = 1.0f / sqrtf((float)c.head_dim);
    const int64_t qd = (int64_t)c.n_q_heads * c.head_dim;
    const ActOut none{nullptr, nullptr}, out_d{rt.act_d.xp, rt.act_d.xs}, out_o{rt.act_o.xp, rt.act_o.xs};
    const ActOperand in_d{rt.act_d.xp, rt.act_d.xs}, in_o{rt.act_o.xp, rt.act_o.xs};
    cudaError_t e;
#define FW(x)                           \
    do {                                \
        e = (x);                        \
        if (e != cudaSuccess) return e; \
    } while (0)
    // embedding rows into the residual stream plus the RoPE table of the rows' positions (the operand and the sums
    // this kernel also writes are replaced by the norm that follows)
    FW(launch_embed_norm(ctx, st, m->embed.qtype, m->embed.data, c.vocab, c.d_model, tokens_dev, token_stride, rows, rt.h,
                         m->layers[0].attn_norm, out_d, rt.ss, rt.cs, rows_dev, c.head_dim, c.rope_theta));
    FW(launch_rmsnorm_rows(ctx, st, rt.h, nullptr, m->layers[0].attn_norm, rt.w_xn, out_d, rows, c.d_model, c.rms_eps));
    for (int L = 0; L < c.n_layers; L++) {
        const LayerW& l = m->layers[L];
        {   // q|k|v over the normed operand; epilogue: f16 rounding, RoPE, q -> buffer, k and v -> cache slots
            EpiArgs a;
            a.ss_in = rt.moe_unit_ss, a.ss_parts = 1, a.d_in = c.d_model, a.eps = 0.f;
            a.kv = rt.kv->view, a.layer = L, a.row_desc = rows_dev, a.cs = rt.cs, a.q_out = rt.q;
            a.n_q_heads = c.n_q_heads, a.n_kv_heads = c.n_kv_heads, a.head_dim = c.head_dim;
            if (l.wv.data) a.n_v_heads = 0;
            FW(launch_gemm_fused(ctx, st, l.wqkv.qtype, l.wqkv.data, l.wqkv.rows, l.wqkv.cols, in_d, rows, EPI_ROPE_STORE, a));
            if (l.wv.data) {
                a.n_q_heads = 0, a.n_kv_heads = 0, a.n_v_heads = c.n_kv_heads;
                FW(launch_gemm_fused(ctx, st, l.wv.qtype, l.wv.data, l.wv.rows, l.wv.cols, in_d, rows, EPI_ROPE_STORE, a));
            }
        }
        FW(launch_attn_decode_rows(ctx, st, rt.kv, L, rt.q, qd, nullptr, out_o, rows_dev, rows, rows_per_seq, c.n_q_heads, scale,
                                   max_len, rt.attn_scratch, s->n_streams * s->max_rows));
        if (comm_world(s->comm) > 1) {
            // tensor-parallel attention: this rank's o_proj holds its heads' columns; the f32 shares are summed over the
            // ranks, then rounded to f16 once, as the single projection is
            FW(launch_gemm_quant(ctx, st, l.wo.qtype, l.wo.data, l.wo.rows, l.wo.cols, in_o, rt.tp_partial, c.d_model, rows, true));
            FW(comm_all_reduce_f32(s->comm, st, rt.tp_partial, (size_t)rows * c.d_model));
            FW(launch_f32_to_f16(ctx, st, rt.tp_partial, rt.w_o, (int64_t)rows * c.d_model));
        } else {
            FW(launch_gemm_quant(ctx, st, l.wo.qtype, l.wo.data, l.wo.rows, l.wo.cols, in_o, rt.w_o, c.d_model, rows, false));
        }
        FW(launch_rmsnorm_rows(ctx, st, rt.h, rt.w_o, l.ffn_norm, rt.w_xn, none, rows, c.d_model, c.rms_eps));
        FW(launch_router_logits(ctx, st, l.router_q, l.router_scale, l.router_bias, rt.w_xn, c.d_model, rows, m->n_experts, c.d_model, rt.moe_logits));
        FW(launch_moe_route(ctx, st, rt.moe_logits, rows, m->n_experts, m->top_k, rt.moe_ids, rt.moe_w));
        FW(launch_moe_ffn(ctx, st, l.experts_qtype, l.experts_gate_up, l.experts_down, m->n_experts, c.d_model, m->moe_ffn, rt.w_xn, c.d_model,
                          rt.moe_zero, rt.moe_ids, rt.moe_w, rows, m->top_k, nullptr, rt.moe_ws, m->expert_lo, m->n_local_experts));
        // sharded experts: every (row, slot) value was computed by exactly one rank, the others hold zero there - the
        // sum over the ranks is exact, and the slot-ordered combine below sees the values of a single GPU
        if (m->n_local_experts > 0)
            FW(comm_all_reduce_f32(s->comm, st, const_cast<float*>(moe_ffn_values(rt.moe_ws, rows, m->top_k, m->n_experts, c.d_model, m->moe_ffn)),
                                   (size_t)rows * m->top_k * c.d_model));
        // the slot-ordered weighted sum (over a zero residual, rounded to f16), its add onto the stream and the next norm
        const void* g = L + 1 < c.n_layers ? (const void*)m->layers[L + 1].attn_norm : (const void*)m->out_norm;
        FW(launch_combine_norm_rows(ctx, st, rt.h, moe_ffn_values(rt.moe_ws, rows, m->top_k, m->n_experts, c.d_model, m->moe_ffn), rt.moe_w,
                                    m->top_k, g, rt.w_xn, out_d, rows, c.d_model, c.rms_eps));
    }
    if (logits) {
        EpiArgs a;
        a.y = logits, a.y_stride = logits_stride, a.y_f32 = 0;
        a.y_every = last_rows_only ? rows_per_seq : 0;
        FW(launch_gemm_fused(ctx, st, m->lm_head.qtype, m->lm_head.data, m->lm_head.rows, m->lm_head.cols, in_d, rows, EPI_PLAIN, a));
    }
#undef FW
    return cudaSuccess;
}

// One forward pass over `rows` rows (rows_per_seq per stream).  Row descriptors and token ids are
// already on the device.  Cursors are not touched here.
static cudaError_t forward_device(tsb_session* s, ModelRt& rt, const int32_t* tokens_dev, int token_stride,
                                  const tsb_row_desc* rows_dev, int rows, int rows_per_seq, int max_len, __half* logits,
                                  int64_t logits_stride, bool last_rows_only = false, int only = PASS_ALL) {
    const bool matmuls_only = only == PASS_MATMULS, skip_matmuls = only == PASS_REST;
    if (rt.model->n_experts > 0)
        return forward_device_moe(s, rt, tokens_dev, token_stride, rows_dev, rows, rows_per_seq, (max_len + 511) / 512 * 512, logits,
                                  logits_stride, last_rows_only);
    if (rt.wide_ok && only == PASS_ALL)
        return forward_device_wide(s, rt, tokens_dev, token_stride, rows_dev, rows, rows_per_seq, (max_len + 511) / 512 * 512, logits,
                                   logits_stride, last_rows_only);
    tsb_ctx* ctx = s->ctx;
    cudaStream_t st = s->stream;
    const tsb_model* m = rt.model;
    const tsb_model_config& c = m->cfg;
    const float scale = 1.0f / sqrtf((float)c.head_dim);
    max_len = (max_len + 511) / 512 * 512;  // the split plan changes only every 512 positions (graph reuse)
    cudaError_t e;
#define FW(x)                         \
    do {                              \
        e = (x);                      \
        if (e != cudaSuccess) return e; \
    } while (0)
    const ActOut out_d{rt.act_d.xp, rt.act_d.xs}, out_o{rt.act_o.xp, rt.act_o.xs}, out_f{rt.act_f.xp, rt.act_f.xs};
    const ActOperand in_d{rt.act_d.xp, rt.act_d.xs}, in_o{rt.act_o.xp, rt.act_o.xs}, in_f{rt.act_f.xp, rt.act_f.xs};
    const int R = s->n_streams * s->max_rows;
    const int parts = c.d_model / 16;
    auto ss_slot = [&](int i) { return rt.ss + (size_t)i * R * parts; };
    // (PASS_MATMULS / PASS_REST: the measurement aids - only the layer matmuls with their real epilogues, or only the
    // other launches of the pass (embedding, attention, head), over whatever the buffers hold)
    // embedding: residual stream, layer 0's operand f16(h * g), sum of h^2 (one partial per row), RoPE table
    if (!matmuls_only) FW(launch_embed_norm(ctx, st, m->embed.qtype, m->embed.data, c.vocab, c.d_model, tokens_dev, token_stride, rows, rt.h,
                         m->layers[0].attn_norm, out_d, ss_slot(0), rt.cs, rows_dev, c.head_dim, c.rope_theta));
    for (int L = 0; L < c.n_layers; L++) {
        const LayerW& l = m->layers[L];
        if (!skip_matmuls) {   // q|k|v matmul; epilogue: 1/rms, RoPE, q -> buffer, k and v -> cache slots
            EpiArgs a;
            a.ss_in = ss_slot(2 * L), a.ss_parts = L == 0 ? 1 : parts, a.d_in = c.d_model, a.eps = c.rms_eps;
            a.kv = rt.kv->view, a.layer = L, a.row_desc = rows_dev, a.cs = rt.cs, a.q_out = rt.q;
            a.n_q_heads = c.n_q_heads, a.n_kv_heads = c.n_kv_heads, a.head_dim = c.head_dim;
            if (l.wv.data) a.n_v_heads = 0;
            FW(launch_gemm_fused(ctx, st, l.wqkv.qtype, l.wqkv.data, l.wqkv.rows, l.wqkv.cols, in_d, rows, EPI_ROPE_STORE, a));
            if (l.wv.data) {  // v in its own block format: the v rows as a second launch, every tile a v tile
                a.n_q_heads = 0, a.n_kv_heads = 0, a.n_v_heads = c.n_kv_heads;
                FW(launch_gemm_fused(ctx, st, l.wv.qtype, l.wv.data, l.wv.rows, l.wv.cols, in_d, rows, EPI_ROPE_STORE, a));
            }
        }
        if (!matmuls_only)
            FW(launch_attn_decode_rows(ctx, st, rt.kv, L, rt.q, (int64_t)c.n_q_heads * c.head_dim, nullptr, out_o, rows_dev, rows,
                                       rows_per_seq, c.n_q_heads, scale, max_len, rt.attn_scratch, s->n_streams * s->max_rows));
        if (skip_matmuls) continue;
        {   // o_proj; epilogue: residual add, next operand f16(h * g_ffn), partial sums of h^2
            EpiArgs a;
            a.h = rt.h, a.g = l.ffn_norm, a.out = out_d, a.ss_out = ss_slot(2 * L + 1);
            FW(launch_gemm_fused(ctx, st, l.wo.qtype, l.wo.data, l.wo.rows, l.wo.cols, in_o, rows, EPI_RESID_NORM, a));
        }
        {   // gate|up matmul; epilogue: 1/rms, SiLU(gate) * up -> operand of the down projection
            EpiArgs a;
            a.ss_in = ss_slot(2 * L + 1), a.ss_parts = parts, a.d_in = c.d_model, a.eps = c.rms_eps, a.out = out_f;
            FW(launch_gemm_fused(ctx, st, l.wgu.qtype, l.wgu.data, l.wgu.rows, l.wgu.cols, in_d, rows, EPI_SILU, a));
        }
        {   // down projection; epilogue: residual add, operand for the next layer's norm (or the final norm)
            EpiArgs a;
            a.h = rt.h, a.g = L + 1 < c.n_layers ? m->layers[L + 1].attn_norm : m->out_norm, a.out = out_d;
            a.ss_out = ss_slot(2 * L + 2);
            FW(launch_gemm_fused(ctx, st, l.wdown.qtype, l.wdown.data, l.wdown.rows, l.wdown.cols, in_f, rows, EPI_RESID_NORM, a));
        }
    }
    if (logits && !matmuls_only) {
        // head over the final-normed operand; row t of the logits sits at logits + t * logits_stride
        EpiArgs a;
        a.ss_in = ss_slot(2 * c.n_layers), a.ss_parts = parts, a.d_in = c.d_model, a.eps = c.rms_eps;
        a.y = logits, a.y_stride = logits_stride, a.y_f32 = 0;
        a.y_every = last_rows_only ? rows_per_seq : 0;  // logits of each stream's last row only, one output row per stream
        FW(launch_gemm_fused(ctx, st, m->lm_head.qtype, m->lm_head.data, m->lm_head.rows, m->lm_head.cols, in_d, rows, EPI_SCALE, a));
    }
#undef FW
    return cudaSuccess;
}

static int32_t blocks_fill_context(tsb_session* s, ModelRt& rt, int stream, int64_t tokens, uint64_t seed) {
    return tsb_kv_fill_random(rt.kv, s->stream, stream, tokens, seed);
}

static cudaError_t blocks_forward(tsb_session* s, ModelRt& rt, const Pass& p) {
    return forward_device(s, rt, p.tokens, p.token_stride, p.rows_dev, p.rows, p.rows_per_seq, p.max_len, (__half*)p.logits.p, p.logits_stride,
                          p.last_rows_only, p.only);
}

const ModelFamily BLOCKS_FAMILY = {
    "block-quantised", false, true, false, blocks_complete, blocks_free_tensors, blocks_weight_bytes, blocks_share, blocks_runtime_init,
    nullptr, blocks_fill_context, blocks_forward,
};

extern "C" {

int32_t tsb_session_time_matmuls(tsb_session* s, int32_t rows, int32_t iters, float* out_ms, int64_t* out_bytes_per_iter,
                                 int32_t* out_launches_per_iter) {
    if (!s || !out_ms) return TSB_ERR_INVALID;
    tsb_ctx* ctx = s->ctx;
    TSB_REQUIRE(ctx, s->target.model->family == &BLOCKS_FAMILY, "the timing covers block-quantised models");
    TSB_REQUIRE(ctx, rows > 0 && rows <= s->n_streams * s->max_rows && iters > 0, "bad rows / iters");
    if (s->target.model->n_experts > 0) return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "the matmul timing covers dense layers only");
    DeviceGuard g(ctx);
    ModelRt& rt = s->target;
    const tsb_model* m = rt.model;
    const tsb_model_config& c = m->cfg;
    const int64_t qkv_dim = (int64_t)(c.n_q_heads + 2 * c.n_kv_heads) * c.head_dim;
    cudaStream_t st = s->stream;
    int64_t bytes = 0;
    int launches = 0;
    // The launches are the pass's own: the same kernels with the same fused epilogues (1/rms + RoPE + K/V store,
    // residual + norm operand, SiLU * up), writing the session's real buffers; the rows sit past every stream's cursor
    // (in-flight slots nobody committed), so the caches' committed contents are untouched.  Attention, embedding and
    // head are left out.
    TSB_REQUIRE(ctx, rows % s->n_streams == 0, "rows must be a whole number of rows per stream");
    const int per = rows / s->n_streams;
    std::vector<int32_t> streams(s->n_streams);
    for (int q = 0; q < s->n_streams; q++) streams[q] = q;
    const tsb_row_desc* rd;
    int max_len;
    s->stage_used = 0;
    int32_t rc = stage_rows(s, rt, streams.data(), s->n_streams, per, nullptr, nullptr, &rd, nullptr, &max_len);
    if (rc) return rc;
    TSB_REQUIRE(ctx, !rt.wide_ok, "the matmul timing covers sessions whose target runs the few-row matmul path (largest pass below %d rows)", WIDE_MIN_ROWS);
    for (int it = -1; it < iters; it++) {  // iteration -1 is a warm-up
        if (it == 0) TSB_CUDA(ctx, cudaEventRecord(s->ev[0], st));
        TSB_CUDA(ctx, forward_device(s, rt, nullptr, 1, rd, rows, per, max_len, nullptr, 0, false, PASS_MATMULS));
    }
    for (const LayerW& l : m->layers) {
        bytes += mat_bytes(l.wqkv) + mat_bytes(l.wv) + mat_bytes(l.wo) + mat_bytes(l.wgu) + mat_bytes(l.wdown);
        launches += (l.wv.data ? 5 : 4) * ((rows + 63) / 64);
    }
    TSB_CUDA(ctx, cudaEventRecord(s->ev[1], st));
    rc = tsb_stream_sync(ctx, st);
    s->stage_used = 0;
    if (rc) return rc;
    TSB_CUDA(ctx, cudaEventElapsedTime(out_ms, s->ev[0], s->ev[1]));
    // activations in and out per launch are part of the algorithmic bytes too
    const int64_t act = (int64_t)rows * 2 * ((int64_t)c.d_model + qkv_dim + (int64_t)c.n_q_heads * c.head_dim + c.d_model + c.d_model +
                                              2 * (int64_t)c.ffn + c.ffn + c.d_model) * c.n_layers;
    if (out_bytes_per_iter) *out_bytes_per_iter = bytes + act;
    if (out_launches_per_iter) *out_launches_per_iter = launches;
    return TSB_OK;
}

int32_t tsb_session_time_pass_rest(tsb_session* s, int32_t rows, int32_t iters, float* out_ms) {
    if (!s || !out_ms) return TSB_ERR_INVALID;
    tsb_ctx* ctx = s->ctx;
    TSB_REQUIRE(ctx, s->target.model->family == &BLOCKS_FAMILY, "the timing covers block-quantised models");
    TSB_REQUIRE(ctx, rows > 0 && rows <= s->n_streams * s->max_rows && iters > 0, "bad rows / iters");
    if (s->target.model->n_experts > 0) return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "the pass timing covers dense layers only");
    DeviceGuard g(ctx);
    ModelRt& rt = s->target;
    TSB_REQUIRE(ctx, rows % s->n_streams == 0, "rows must be a whole number of rows per stream");
    TSB_REQUIRE(ctx, !rt.wide_ok, "the pass timing covers sessions whose target runs the few-row matmul path (largest pass below %d rows)", WIDE_MIN_ROWS);
    const int per = rows / s->n_streams;
    std::vector<int32_t> streams(s->n_streams), toks(rows, 0);
    for (int q = 0; q < s->n_streams; q++) streams[q] = q;
    const tsb_row_desc* rd;
    const int32_t* td;
    int max_len;
    s->stage_used = 0;
    int32_t rc = stage_rows(s, rt, streams.data(), s->n_streams, per, nullptr, toks.data(), &rd, &td, &max_len);
    if (rc) return rc;
    cudaStream_t st = s->stream;
    for (int it = -1; it < iters; it++) {  // iteration -1 is a warm-up
        if (it == 0) TSB_CUDA(ctx, cudaEventRecord(s->ev[0], st));
        TSB_CUDA(ctx, forward_device(s, rt, td, 1, rd, rows, per, max_len, (__half*)s->logits_target.p, rt.model->cfg.vocab, false, PASS_REST));
    }
    TSB_CUDA(ctx, cudaEventRecord(s->ev[1], st));
    rc = tsb_stream_sync(ctx, st);
    s->stage_used = 0;
    if (rc) return rc;
    TSB_CUDA(ctx, cudaEventElapsedTime(out_ms, s->ev[0], s->ev[1]));
    return TSB_OK;
}

}  // extern "C"
