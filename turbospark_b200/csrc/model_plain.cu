// The plain-weight decoder family (tsb_model_create_plain): models, session buffers, forward pass.
//
// A layer is four launches, plus the embedding before the first and norm + head after the last:
//   norm + token shift           f32 residual stream -> the mixer's input and the feed-forward's input
//   input matmul                 one packed matrix over queries | keys | head gates | gate-up pairs; its epilogue stores the
//                                queries, writes the keys into their cache slots, keeps the gates in f32 and leaves
//                                act(gate) * up beside the attention output
//   window attention             over the key-only cache, gate applied where a head's output is finished
//   output matmul                [W_o | W_down] over [heads | feed-forward]: the two sublayers of a parallel layer add up
//                                inside one product, whose epilogue adds it to the stream
#include <algorithm>
#include <cstring>
#include <new>

#include "model_plain.cuh"

namespace {

__device__ __forceinline__ uint32_t mix32(uint32_t x) {
    x ^= x >> 16;
    x *= 0x7feb352du;
    x ^= x >> 15;
    x *= 0x846ca68bu;
    x ^= x >> 16;
    return x;
}
// uniform in +-amp around mid, zero in the padding columns
template <typename T>
__global__ void fill_plain_kernel(T* p, int64_t rows, int64_t cols, int64_t valid_cols, float mid, float amp, uint32_t seed) {
    const int64_t n = rows * cols;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
        const uint32_t h = mix32((uint32_t)i * 0x9E3779B9u + seed) ^ mix32((uint32_t)(i >> 32) + seed * 31u);
        const float u = (float)(h >> 8) * (1.0f / 16777216.0f) * 2.f - 1.f;
        p[i] = (T)(i % cols < valid_cols ? mid + amp * u : 0.f);
    }
}

int32_t zeroed(tsb_ctx* ctx, size_t bytes, void** out) {
    int32_t rc = tsb_alloc(ctx, bytes, out);
    if (rc) return rc;
    TSB_CUDA(ctx, cudaMemset(*out, 0, bytes));
    return TSB_OK;
}

float bf16_to_f(uint16_t b) {
    const uint32_t u = (uint32_t)b << 16;
    float f;
    memcpy(&f, &u, 4);
    return f;
}

// host tensor -> the model's element type
void convert(const void* host, int host_type, int64_t n, bool f32, std::vector<uint8_t>& out) {
    out.resize((size_t)n * (f32 ? 4 : 2));
    if (host_type == (f32 ? TSB_F32 : TSB_BF16)) {
        memcpy(out.data(), host, out.size());
    } else if (f32) {
        const uint16_t* s = static_cast<const uint16_t*>(host);
        float* d = reinterpret_cast<float*>(out.data());
        for (int64_t i = 0; i < n; i++) d[i] = bf16_to_f(s[i]);
    } else {
        const float* s = static_cast<const float*>(host);
        __nv_bfloat16* d = reinterpret_cast<__nv_bfloat16*>(out.data());
        for (int64_t i = 0; i < n; i++) d[i] = __float2bfloat16_rn(s[i]);
    }
}

int32_t plain_complete(const tsb_model* tm) {
    tsb_ctx* ctx = tm->ctx;
    const PlainModel* m = tm->plain;
    const uint32_t want = 1u << TSB_P_EMBED | 1u << TSB_P_HEAD | 1u << TSB_P_FINAL_NORM;
    TSB_REQUIRE(ctx, (m->set & want) == want, "embedding, head or final norm missing");
    for (size_t i = 0; i < m->layers.size(); i++) {
        const PlainLayer& l = m->layers[i];
        uint32_t w = 1u << TSB_P_NORM | 1u << TSB_P_Q | 1u << TSB_P_K | 1u << TSB_P_O;
        if (l.cfg.token_shift) w |= 1u << TSB_P_SHIFT;
        if (l.cfg.head_gate) w |= 1u << TSB_P_HEAD_GATE;
        if (l.cfg.log_bias) w |= 1u << TSB_P_R1 | 1u << TSB_P_R2;
        if (l.cfg.ffn > 0) w |= 1u << TSB_P_FF_GATE | 1u << TSB_P_FF_UP | 1u << TSB_P_FF_DOWN;
        TSB_REQUIRE(ctx, (l.set & w) == w, "layer %zu is missing a tensor (have %x, need %x)", i, l.set, w);
    }
    return TSB_OK;
}

void plain_free(tsb_model* tm) {
    PlainModel* m = tm->plain;
    if (!m) return;
    tsb_ctx* ctx = tm->ctx;
    for (PlainLayer& l : m->layers)
        if (l.owned)
            for (void* p : {l.in.data, l.out.data, (void*)l.gain, (void*)l.mu, (void*)l.r1, (void*)l.r2})
                if (p) tsb_free(ctx, p);
    if (m->owned)
        for (void* p : {m->head.data, m->embed, (void*)m->final_gain})
            if (p) tsb_free(ctx, p);
    delete m;
    tm->plain = nullptr;
}

// bytes a pass reads of the matrices (the embedding is read by rows and not counted)
int64_t plain_weight_bytes(const tsb_model* tm) {
    const PlainModel* m = tm->plain;
    int64_t n = (int64_t)m->cfg.vocab * m->cfg.d_model;
    for (const PlainLayer& l : m->layers) {
        const tsb_plain_layer& c = l.cfg;
        n += (int64_t)m->cfg.d_model * ((int64_t)c.head_dim * (2 * c.n_q_heads + c.n_kv_heads) + (c.head_gate ? c.n_q_heads : 0) + 3 * (int64_t)c.ffn);
    }
    return n * m->elem;
}

int32_t plain_share(tsb_model* dt, int32_t dst_layer, const tsb_model* st, int32_t src_layer) {
    tsb_ctx* ctx = dt->ctx;
    PlainModel* d = dt->plain;
    const PlainModel* s = st->plain;
    TSB_REQUIRE(ctx, d->cfg.d_model == s->cfg.d_model && d->cfg.vocab == s->cfg.vocab && d->f32 == s->f32, "models differ in width, vocabulary or type");
    if (dst_layer < 0) {
        if (d->owned)
            for (void* p : {d->head.data, d->embed, (void*)d->final_gain})
                if (p) tsb_free(ctx, p);
        d->head = s->head, d->embed = s->embed, d->final_gain = s->final_gain, d->set = s->set, d->owned = false;
        return TSB_OK;
    }
    TSB_REQUIRE(ctx, dst_layer < d->cfg.n_layers && src_layer >= 0 && src_layer < s->cfg.n_layers, "layer out of range");
    PlainLayer& l = d->layers[dst_layer];
    TSB_REQUIRE(ctx, memcmp(&l.cfg, &s->layers[src_layer].cfg, sizeof l.cfg) == 0, "layer shapes differ");
    if (l.owned)
        for (void* p : {l.in.data, l.out.data, (void*)l.gain, (void*)l.mu, (void*)l.r1, (void*)l.r2})
            if (p) tsb_free(ctx, p);
    l = s->layers[src_layer];
    l.owned = false;
    return TSB_OK;
}

void plain_runtime_free(ModelRt& rt) {
    delete rt.plain;  // the device buffers belong to the session
    rt.plain = nullptr;
}

int32_t plain_runtime_init(tsb_session* s, ModelRt& rt, const tsb_model* tm, const SessionShape& shape, bool is_draft) {
    (void)is_draft;
    tsb_ctx* ctx = s->ctx;
    const PlainModel* m = tm->plain;
    rt.model = tm;
    std::vector<int32_t> heads, dims;
    for (const PlainLayer& l : m->layers) heads.push_back(l.cfg.n_kv_heads), dims.push_back(l.head_pad);
    int32_t rc = kv_create_keys(ctx, m->cfg.n_layers, heads.data(), dims.data(), m->elem, shape.page_tokens, shape.num_pages, shape.n_streams,
                                shape.pages_per_seq, &rt.kv);
    if (rc) return rc;
    PlainRt* p = rt.plain = new (std::nothrow) PlainRt();
    if (!p) return TSB_ERR_OOM;
    // matmul operands are read in whole token tiles
    p->rows = (int)plain_pad(std::max(shape.pass_rows, 32), 32);
    p->in_stride = m->d_pad;
    for (const PlainLayer& l : m->layers) {
        p->q_stride = std::max<int64_t>(p->q_stride, l.q_rows);
        p->cat_stride = std::max<int64_t>(p->cat_stride, l.out.cols);
        p->gate_stride = std::max(p->gate_stride, l.cfg.n_q_heads);
    }
    p->fin_rows = (int)plain_pad(std::max(std::max(shape.n_streams * shape.max_rows, std::min(shape.pass_rows, 256)), 32), 32);
    auto A = [&](size_t bytes, void** q) {
        int32_t r = dev_alloc(ctx, s->owned, bytes, q);
        if (r == TSB_OK && cudaMemset(*q, 0, bytes) != cudaSuccess) r = tsb_fail(ctx, TSB_ERR_CUDA, "clearing a work buffer failed");
        return r;
    };
    const size_t R = p->rows, e = m->elem;
    if ((rc = A(R * m->cfg.d_model * 4, (void**)&p->x)) || (rc = A(R * p->in_stride * e, &p->mix)) || (rc = A(R * p->in_stride * e, &p->h)) ||
        (rc = A(R * p->q_stride * e, &p->q)) || (rc = A(R * p->cat_stride * e, &p->cat)) || (rc = A(R * p->gate_stride * 4, (void**)&p->gate)) ||
        (rc = A((size_t)p->fin_rows * p->in_stride * e, &p->fin)) || (rc = A(plain_gemm_workspace_bytes(ctx), &p->gemm_ws)) ||
        (rc = A(wattn_scratch_bytes(ctx), &p->attn_ws)))
        return rc;
    if (m->any_shift) {
        ShiftState& st = p->shift;
        st.width = m->cfg.d_model, st.n_streams = shape.n_streams;
        st.ring_rows = 4;
        while (st.ring_rows < shape.max_rows + 2) st.ring_rows *= 2;
        const size_t per = (size_t)m->cfg.n_layers * shape.n_streams * m->cfg.d_model * 4;
        if ((rc = A(per * st.ring_rows, (void**)&st.ring)) || (rc = A(per, (void**)&st.before))) return rc;
        rt.kv->state_ring = st.ring_rows;
    }
    rt.fed.assign(shape.n_streams, std::vector<int32_t>());
    rt.pending.assign(shape.n_streams, PendingVerify());
    return TSB_OK;
}

int32_t plain_fill_context(tsb_session* s, ModelRt& rt, int stream, int64_t tokens, uint64_t seed) {
    return kv_fill_keys(rt.kv, s->stream, stream, tokens, seed);  // the shift state keeps what it holds
}

// The query tiles of a ragged pass for one group size: few-query tiles hold a whole stream's rows.
struct TileLists {
    int group = 0, rows_per_tile = 0;
    AttnBatch batch;
};

cudaError_t plain_forward(tsb_session* s, ModelRt& rt, const Pass& p) {
    tsb_ctx* ctx = s->ctx;
    cudaStream_t st = s->stream;
    const PlainModel* m = rt.model->plain;
    PlainRt* b = rt.plain;
    const int d = m->cfg.d_model;
    cudaError_t e;
#define FW(x)                           \
    do {                                \
        e = (x);                        \
        if (e != cudaSuccess) return e; \
    } while (0)
    const int max_len = (p.max_len + 511) / 512 * 512;  // the split plan changes only every 512 positions (graph reuse)
    std::vector<TileLists> lists;
    int longest = p.rows_per_seq;
    if (p.rows_per_seq == 0) {
        for (int i = 0; i < p.n_groups; i++) longest = std::max(longest, p.groups[i].n_rows);
        for (const PlainLayer& l : m->layers) {
            const int grp = l.cfg.n_q_heads / l.cfg.n_kv_heads;
            const int rpt = wattn_rows_per_tile(l.head_pad, grp);
            bool have = m->f32;  // the f32 kernel takes rows one by one
            for (const TileLists& t : lists) have |= t.group == grp && t.rows_per_tile == rpt;
            if (have) continue;
            std::vector<AttnTile> small, large;
            TileLists t;
            t.group = grp, t.rows_per_tile = rpt;
            for (int i = 0; i < p.n_groups; i++) {
                const RowGroup& g = p.groups[i];
                if (g.n_rows * grp <= WATTN_SMALL_Q) {
                    small.push_back({g.first_row, g.n_rows});
                    t.batch.small_queries = std::max(t.batch.small_queries, g.n_rows * grp);
                } else {
                    for (int r = 0; r < g.n_rows; r += rpt) large.push_back({g.first_row + r, std::min(rpt, g.n_rows - r)});
                }
            }
            t.batch.n_small = (int)small.size(), t.batch.n_large = (int)large.size();
            small.insert(small.end(), large.begin(), large.end());
            const int32_t* dev = nullptr;
            if (session_stage_ints(s, reinterpret_cast<const int32_t*>(small.data()), (int)small.size() * 2, &dev) != TSB_OK) return cudaErrorMemoryAllocation;
            t.batch.small = reinterpret_cast<const AttnTile*>(dev), t.batch.large = t.batch.small + t.batch.n_small;
            lists.push_back(t);
        }
    }
    const bool use_before = m->any_shift && longest >= b->shift.ring_rows;
    FW(launch_plain_embed(ctx, st, m->f32, m->embed, m->cfg.vocab, d, p.tokens, p.token_stride, p.rows, b->x));
    if (use_before) FW(launch_shift_before(ctx, st, b->shift, m->cfg.n_layers, p.rows_dev, p.rows));
    for (int L = 0; L < m->cfg.n_layers; L++) {
        const PlainLayer& l = m->layers[L];
        const tsb_plain_layer& c = l.cfg;
        FW(launch_norm_shift(ctx, st, m->f32, b->x, d, l.gain, m->cfg.norm_eps, c.token_shift ? l.mu : nullptr, p.rows_dev, p.rows, b->shift, L, use_before,
                             b->mix, c.ffn > 0 ? b->h : nullptr, b->in_stride));
        const int64_t cat_stride = l.out.cols;
        PlainEpi in;
        in.kind = PLAIN_MIXER;
        in.q = b->q, in.q_stride = l.q_rows, in.q_rows = l.q_rows, in.k_rows = l.k_rows;
        in.keys = rt.kv->key_layers[L], in.rows = p.rows_dev;
        in.gate = b->gate, in.gate_rows = c.head_gate ? c.n_q_heads : 0;
        if (c.ffn > 0) {
            in.pair_row0 = (int)(l.in.rows - 2 * l.ffn_pad), in.n_pairs = l.ffn_pad, in.act = c.act;
            in.a = static_cast<uint8_t*>(b->cat) + (size_t)l.o_cols * m->elem, in.a_stride = cat_stride;
        }
        FW(launch_plain_gemm(ctx, st, m->f32, l.in, b->mix, b->h, b->in_stride, b->rows, p.rows, in, b->gemm_ws));
        WindowAttn a;
        a.keys = rt.kv->key_layers[L], a.q = b->q, a.q_stride = l.q_rows;
        a.gate = c.head_gate ? b->gate : nullptr, a.out = b->cat, a.out_stride = cat_stride, a.rows = p.rows_dev;
        a.n_q_heads = c.n_q_heads, a.scale = c.score_scale, a.cap = c.score_cap, a.window = c.window;
        if (c.log_bias) a.r1 = l.r1, a.r2 = l.r2;
        AttnBatch batch;
        for (const TileLists& t : lists)
            if (t.group == c.n_q_heads / c.n_kv_heads && t.rows_per_tile == wattn_rows_per_tile(l.head_pad, t.group)) batch = t.batch;
        batch.rows = p.rows, batch.rows_per_seq = p.rows_per_seq, batch.max_len = max_len;
        FW(launch_window_attn(ctx, st, m->f32, a, batch, b->attn_ws));
        PlainEpi out;
        out.kind = PLAIN_ADD, out.y = b->x, out.y_stride = d, out.n_valid = d;
        FW(launch_plain_gemm(ctx, st, m->f32, l.out, b->cat, nullptr, cat_stride, b->rows, p.rows, out, b->gemm_ws));
    }
    if (p.logits) {
        const bool last = p.last_rows_only && p.rows_per_seq > 1;
        const int n = p.rows_per_seq == 0 ? p.n_want : last ? p.rows / p.rows_per_seq : p.rows;
        if (n > 0) {
            FW(launch_norm_rows(ctx, st, m->f32, b->x, d, m->final_gain, m->cfg.norm_eps, p.rows_per_seq == 0 ? p.want_dev : nullptr,
                                last ? p.rows_per_seq - 1 : 0, last ? p.rows_per_seq : 1, n, b->fin, b->in_stride));
            PlainEpi hd;
            hd.kind = PLAIN_STORE, hd.y = static_cast<float*>(p.logits.p), hd.y_stride = p.logits_stride, hd.n_valid = m->cfg.vocab, hd.cap = m->cfg.logit_cap;
            FW(launch_plain_gemm(ctx, st, m->f32, m->head, b->fin, nullptr, b->in_stride, b->fin_rows, n, hd, b->gemm_ws));
        }
    }
#undef FW
    return cudaSuccess;
}

const ModelFamily PLAIN_FAMILY = {
    "plain-weight", true, false, true, plain_complete, plain_free, plain_weight_bytes, plain_share, plain_runtime_init,
    plain_runtime_free, plain_fill_context, plain_forward,
};

}  // namespace

extern "C" {

int32_t tsb_model_create_plain(tsb_ctx* ctx, const tsb_plain_config* cfg, const tsb_plain_layer* layers, tsb_model** out) {
    if (!ctx || !cfg || !layers || !out) return TSB_ERR_INVALID;
    *out = nullptr;
    TSB_REQUIRE(ctx, cfg->n_layers > 0 && cfg->d_model > 0 && cfg->vocab > 0 && cfg->max_context > 0, "model dimensions must be positive");
    TSB_REQUIRE(ctx, cfg->compute == TSB_BF16 || cfg->compute == TSB_F32, "compute must be TSB_BF16 or TSB_F32");
    TSB_REQUIRE(ctx, cfg->norm_eps >= 0.f, "norm_eps must not be negative");
    const bool f32 = cfg->compute == TSB_F32;
    for (int i = 0; i < cfg->n_layers; i++) {
        const tsb_plain_layer& l = layers[i];
        TSB_REQUIRE(ctx, l.n_q_heads > 0 && l.n_kv_heads > 0 && l.head_dim > 0 && l.n_q_heads % l.n_kv_heads == 0,
                    "layer %d: query heads must be a positive multiple of the key heads", i);
        TSB_REQUIRE(ctx, l.window >= 0 && l.ffn >= 0, "layer %d: window and ffn must not be negative", i);
        TSB_REQUIRE(ctx, l.act == TSB_ACT_GELU_TANH || l.act == TSB_ACT_SILU, "layer %d: unknown activation", i);
        if (!wattn_supported(l.head_dim, l.n_q_heads / l.n_kv_heads, f32))
            return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "layer %d: head size %d with %d query heads per key head is outside the attention kernels", i, l.head_dim,
                            l.n_q_heads / l.n_kv_heads);
    }
    tsb_model* tm = new (std::nothrow) tsb_model();
    PlainModel* m = new (std::nothrow) PlainModel();
    if (!tm || !m) {
        delete tm;
        delete m;
        return TSB_ERR_OOM;
    }
    tm->ctx = ctx, tm->family = &PLAIN_FAMILY, tm->plain = m;
    // what the session and the samplers read of a model
    tm->cfg.n_layers = cfg->n_layers, tm->cfg.d_model = cfg->d_model, tm->cfg.vocab = cfg->vocab, tm->cfg.max_context = cfg->max_context;
    tm->cfg.n_q_heads = layers[0].n_q_heads, tm->cfg.n_kv_heads = layers[0].n_kv_heads, tm->cfg.head_dim = layers[0].head_dim, tm->cfg.ffn = layers[0].ffn;
    tm->cfg.rms_eps = cfg->norm_eps;
    m->cfg = *cfg, m->f32 = f32, m->elem = f32 ? 4 : 2;
    m->d_pad = plain_pad(cfg->d_model, PLAIN_COL_PAD);
    m->head.rows = plain_pad(cfg->vocab, PLAIN_ROW_PAD), m->head.cols = m->d_pad;
    m->layers.resize(cfg->n_layers);
    for (int i = 0; i < cfg->n_layers; i++) {
        PlainLayer& l = m->layers[i];
        l.cfg = layers[i];
        m->any_shift |= l.cfg.token_shift != 0;
        l.head_pad = wattn_pad_dim(l.cfg.head_dim, f32);
        l.q_rows = l.cfg.n_q_heads * l.head_pad, l.k_rows = l.cfg.n_kv_heads * l.head_pad;
        l.ffn_pad = (int)plain_pad(l.cfg.ffn, 64);
        l.in.rows = plain_pad(l.q_rows + l.k_rows + (l.cfg.head_gate ? l.cfg.n_q_heads : 0), PLAIN_ROW_PAD) + 2 * l.ffn_pad;
        l.in.cols = m->d_pad;
        l.o_cols = (int)plain_pad(l.q_rows, PLAIN_COL_PAD);
        l.out.rows = plain_pad(cfg->d_model, PLAIN_ROW_PAD), l.out.cols = l.o_cols + l.ffn_pad;
    }
    *out = tm;
    return TSB_OK;
}

int32_t tsb_model_set_plain(tsb_model* tm, int32_t layer, int32_t which, int32_t host_type, const void* host, int64_t rows, int64_t cols) {
    if (!tm) return TSB_ERR_INVALID;
    tsb_ctx* ctx = tm->ctx;
    TSB_REQUIRE(ctx, tm->family == &PLAIN_FAMILY, "the model does not hold plain tensors");
    TSB_REQUIRE(ctx, host && (host_type == TSB_BF16 || host_type == TSB_F32), "null data or unknown host type");
    PlainModel* m = tm->plain;
    const int64_t d = m->cfg.d_model, V = m->cfg.vocab;
    PlainLayer* l = nullptr;
    if (which >= TSB_P_NORM) {
        TSB_REQUIRE(ctx, layer >= 0 && layer < m->cfg.n_layers, "layer %d outside the model", layer);
        l = &m->layers[layer];
    }
    const tsb_plain_layer c = l ? l->cfg : tsb_plain_layer{};
    const int64_t H = c.n_q_heads, G = c.n_kv_heads, D = c.head_dim, F = c.ffn;
    int64_t wr = 1, wc = 1;
    switch (which) {
        case TSB_P_EMBED: case TSB_P_HEAD: wr = V, wc = d; break;
        case TSB_P_FINAL_NORM: case TSB_P_NORM: break;
        case TSB_P_SHIFT: wc = c.token_shift ? d : -1; break;
        case TSB_P_Q: wr = H * D, wc = d; break;
        case TSB_P_K: wr = G * D, wc = d; break;
        case TSB_P_HEAD_GATE: wr = c.head_gate ? H : -1, wc = d; break;
        case TSB_P_R1: case TSB_P_R2: wc = c.log_bias ? H : -1; break;
        case TSB_P_O: wr = d, wc = H * D; break;
        case TSB_P_FF_GATE: case TSB_P_FF_UP: wr = F > 0 ? F : -1, wc = d; break;
        case TSB_P_FF_DOWN: wr = d, wc = F > 0 ? F : -1; break;
        default: return tsb_fail(ctx, TSB_ERR_INVALID, "no such tensor (%d)", which);
    }
    TSB_REQUIRE(ctx, wr > 0 && wc > 0, "layer %d has no tensor %d", layer, which);
    TSB_REQUIRE(ctx, rows == wr && cols == wc, "tensor %d of layer %d must be %lld x %lld, got %lld x %lld", which, layer, (long long)wr, (long long)wc,
                (long long)rows, (long long)cols);
    DeviceGuard g(ctx);
    int32_t rc;
    std::vector<uint8_t> v;
    // small f32 vectors
    float** vec = which == TSB_P_FINAL_NORM ? &m->final_gain : which == TSB_P_NORM ? &l->gain : which == TSB_P_SHIFT ? &l->mu
                : which == TSB_P_R1 ? &l->r1 : which == TSB_P_R2 ? &l->r2 : nullptr;
    uint32_t& set = l ? l->set : m->set;
    if (vec) {
        convert(host, host_type, wc, true, v);
        if (!*vec && (rc = tsb_alloc(ctx, (size_t)wc * 4, (void**)vec))) return rc;
        TSB_CUDA(ctx, cudaMemcpy(*vec, v.data(), v.size(), cudaMemcpyHostToDevice));
        set |= 1u << which;
        return TSB_OK;
    }
    const size_t es = m->elem;
    convert(host, host_type, wr * wc, m->f32, v);
    if (which == TSB_P_EMBED) {
        if (!m->embed && (rc = tsb_alloc(ctx, v.size(), &m->embed))) return rc;
        TSB_CUDA(ctx, cudaMemcpy(m->embed, v.data(), v.size(), cudaMemcpyHostToDevice));
        set |= 1u << which;
        return TSB_OK;
    }
    PlainMat& mat = which == TSB_P_HEAD ? m->head : which == TSB_P_O || which == TSB_P_FF_DOWN ? l->out : l->in;
    if (!mat.data && (rc = zeroed(ctx, (size_t)mat.rows * mat.cols * es, &mat.data))) return rc;
    uint8_t* base = static_cast<uint8_t*>(mat.data);
    const size_t pitch = (size_t)mat.cols * es;
    // block of n_rows x n_cols of the host tensor at (hr, hc) -> the packed matrix at (dr, dc)
    auto put = [&](int64_t dr, int64_t dc, int64_t hr, int64_t hc, int64_t n_rows, int64_t n_cols) {
        return cudaMemcpy2D(base + (size_t)dr * pitch + (size_t)dc * es, pitch, v.data() + ((size_t)hr * wc + hc) * es, (size_t)wc * es, (size_t)n_cols * es,
                            (size_t)n_rows, cudaMemcpyHostToDevice);
    };
    switch (which) {
        case TSB_P_HEAD: TSB_CUDA(ctx, put(0, 0, 0, 0, wr, wc)); break;
        case TSB_P_Q:
            for (int64_t h = 0; h < H; h++) TSB_CUDA(ctx, put(h * l->head_pad, 0, h * D, 0, D, d));
            break;
        case TSB_P_K:
            for (int64_t h = 0; h < G; h++) TSB_CUDA(ctx, put(l->q_rows + h * l->head_pad, 0, h * D, 0, D, d));
            break;
        case TSB_P_HEAD_GATE: TSB_CUDA(ctx, put(l->q_rows + l->k_rows, 0, 0, 0, H, d)); break;
        case TSB_P_O:
            for (int64_t h = 0; h < H; h++) TSB_CUDA(ctx, put(0, h * l->head_pad, 0, h * D, d, D));
            break;
        case TSB_P_FF_GATE: case TSB_P_FF_UP: {
            const int64_t row0 = mat.rows - 2 * l->ffn_pad + (which == TSB_P_FF_UP ? 8 : 0);
            for (int64_t i = 0; i < F; i += 8) TSB_CUDA(ctx, put(row0 + 2 * i, 0, i, 0, std::min<int64_t>(8, F - i), d));
            break;
        }
        case TSB_P_FF_DOWN: TSB_CUDA(ctx, put(0, l->o_cols, 0, 0, d, F)); break;
    }
    set |= 1u << which;
    return TSB_OK;
}

int32_t tsb_model_fill_plain(tsb_model* tm, uint64_t seed) {
    if (!tm) return TSB_ERR_INVALID;
    tsb_ctx* ctx = tm->ctx;
    TSB_REQUIRE(ctx, tm->family == &PLAIN_FAMILY, "the model does not hold plain tensors");
    PlainModel* m = tm->plain;
    DeviceGuard g(ctx);
    uint32_t sd = (uint32_t)seed * 2654435761u + (uint32_t)(seed >> 32) + 1u;
    int32_t rc = TSB_OK;
    auto fill = [&](void** p, bool f32, int64_t rows, int64_t cols, int64_t valid, float mid, float amp) {
        if (rc) return;
        if (!*p && (rc = tsb_alloc(ctx, (size_t)rows * cols * (f32 ? 4 : 2), p))) return;
        if (f32) fill_plain_kernel<float><<<1024, 256>>>((float*)*p, rows, cols, valid, mid, amp, sd);
        else fill_plain_kernel<__nv_bfloat16><<<1024, 256>>>((__nv_bfloat16*)*p, rows, cols, valid, mid, amp, sd);
        sd = sd * 1664525u + 1013904223u;
    };
    const int64_t d = m->cfg.d_model;
    const float a_in = sqrtf(3.f / (float)d);
    fill(&m->embed, m->f32, m->cfg.vocab, d, d, 0.f, 1.7f);
    fill(&m->head.data, m->f32, m->head.rows, m->head.cols, d, 0.f, a_in);
    fill((void**)&m->final_gain, true, 1, 1, 1, 1.f, 0.f);
    m->set = ~0u;
    for (PlainLayer& l : m->layers) {
        fill(&l.in.data, m->f32, l.in.rows, l.in.cols, d, 0.f, a_in);
        fill(&l.out.data, m->f32, l.out.rows, l.out.cols, l.out.cols, 0.f, 0.5f * sqrtf(3.f / (float)l.out.cols));
        fill((void**)&l.gain, true, 1, 1, 1, 1.f, 0.f);
        fill((void**)&l.mu, true, 1, d, d, 0.5f, 0.4f);
        fill((void**)&l.r1, true, 1, l.cfg.n_q_heads, l.cfg.n_q_heads, 1.f, 0.5f);
        fill((void**)&l.r2, true, 1, l.cfg.n_q_heads, l.cfg.n_q_heads, 0.3f, 0.2f);
        l.set = ~0u;
    }
    if (rc) return rc;
    TSB_CUDA(ctx, cudaDeviceSynchronize());
    return TSB_OK;
}

// ---- the mechanisms as operators

size_t tsb_plain_gemm_workspace_bytes(const tsb_ctx* ctx) { return ctx ? plain_gemm_workspace_bytes(ctx) : 0; }
size_t tsb_window_attention_scratch_bytes(const tsb_ctx* ctx) { return ctx ? wattn_scratch_bytes(ctx) : 0; }

static int32_t check_gemm(tsb_ctx* ctx, int32_t type, const void* w, int64_t rows, int64_t cols, const void* x, int32_t x_rows, int32_t tokens, void* ws) {
    TSB_REQUIRE(ctx, w && x && ws && (type == TSB_BF16 || type == TSB_F32), "null buffer or unknown type");
    TSB_REQUIRE(ctx, rows > 0 && rows % PLAIN_ROW_PAD == 0 && cols > 0 && cols % PLAIN_COL_PAD == 0, "rows must be a multiple of %d and cols of %d",
                PLAIN_ROW_PAD, PLAIN_COL_PAD);
    TSB_REQUIRE(ctx, tokens > 0 && x_rows >= 32 && x_rows >= tokens, "x needs at least max(32, tokens) allocated rows");
    TSB_REQUIRE(ctx, (uintptr_t)w % 16 == 0 && (uintptr_t)x % 16 == 0, "w and x must be 16-byte aligned");
    return TSB_OK;
}

int32_t tsb_plain_gemm(tsb_ctx* ctx, tsb_stream s, int32_t type, const void* w, int64_t rows, int64_t cols, const void* x, int32_t x_rows, int32_t tokens,
                       float* y, int64_t y_stride, int32_t n_valid, float cap, int32_t add, void* workspace) {
    if (!ctx) return TSB_ERR_INVALID;
    int32_t rc = check_gemm(ctx, type, w, rows, cols, x, x_rows, tokens, workspace);
    if (rc) return rc;
    TSB_REQUIRE(ctx, y && n_valid > 0 && n_valid <= rows && y_stride >= n_valid, "bad output");
    DeviceGuard g(ctx);
    PlainEpi e;
    e.kind = add ? PLAIN_ADD : PLAIN_STORE, e.y = y, e.y_stride = y_stride, e.n_valid = n_valid, e.cap = cap;
    TSB_CUDA(ctx, launch_plain_gemm(ctx, (cudaStream_t)s, type == TSB_F32, PlainMat{const_cast<void*>(w), rows, cols}, x, nullptr, cols, x_rows, tokens, e,
                                    workspace));
    return TSB_OK;
}

int32_t tsb_plain_gemm_pairs(tsb_ctx* ctx, tsb_stream s, int32_t type, const void* w, int64_t rows, int64_t cols, const void* x, int32_t x_rows,
                             int32_t tokens, void* a, int64_t a_stride, int32_t n_pairs, int32_t act, void* workspace) {
    if (!ctx) return TSB_ERR_INVALID;
    int32_t rc = check_gemm(ctx, type, w, rows, cols, x, x_rows, tokens, workspace);
    if (rc) return rc;
    TSB_REQUIRE(ctx, a && n_pairs > 0 && 2 * (int64_t)n_pairs <= rows && a_stride >= n_pairs, "bad output");
    TSB_REQUIRE(ctx, act == TSB_ACT_GELU_TANH || act == TSB_ACT_SILU, "unknown activation");
    DeviceGuard g(ctx);
    PlainEpi e;
    e.kind = PLAIN_MIXER, e.pair_row0 = 0, e.n_pairs = n_pairs, e.act = act, e.a = a, e.a_stride = a_stride;
    TSB_CUDA(ctx, launch_plain_gemm(ctx, (cudaStream_t)s, type == TSB_F32, PlainMat{const_cast<void*>(w), rows, cols}, x, x, cols, x_rows, tokens, e,
                                    workspace));
    return TSB_OK;
}

int32_t tsb_norm_shift_rows(tsb_ctx* ctx, tsb_stream s, int32_t type, const float* x, int32_t d, const float* gain, float eps, const float* mu,
                            const tsb_row_desc* rows_dev, int32_t rows, float* state, int32_t n_streams, int32_t ring, void* mix_out, void* h_out,
                            int64_t out_stride) {
    if (!ctx) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, x && gain && rows_dev && mix_out && d > 0 && rows > 0 && out_stride >= d && (type == TSB_BF16 || type == TSB_F32), "bad arguments");
    TSB_REQUIRE(ctx, (uintptr_t)x % 16 == 0 && (uintptr_t)mu % 16 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)mix_out % 16 == 0 && (uintptr_t)h_out % 16 == 0,
                "buffers must be 16-byte aligned");
    TSB_REQUIRE(ctx, !mu || (state && n_streams > 0 && ring >= 2 && (ring & (ring - 1)) == 0), "a shift needs its state, ring a power of two");
    DeviceGuard g(ctx);
    ShiftState st;
    st.ring = state, st.width = d, st.ring_rows = ring, st.n_streams = n_streams;
    TSB_CUDA(ctx, launch_norm_shift(ctx, (cudaStream_t)s, type == TSB_F32, x, d, gain, eps, mu, rows_dev, rows, st, 0, false, mix_out, h_out, out_stride));
    return TSB_OK;
}

int32_t tsb_kv_create_keys(tsb_ctx* ctx, int32_t type, int32_t layers, int32_t kv_heads, int32_t head_dim, int32_t page_tokens, int32_t num_pages,
                           int32_t max_seqs, int32_t max_pages_per_seq, tsb_kv** out) {
    if (!ctx || !out) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, (type == TSB_BF16 || type == TSB_F32) && layers > 0 && kv_heads > 0, "unknown type or bad sizes");
    TSB_REQUIRE(ctx, wattn_pad_dim(head_dim, type == TSB_F32) == head_dim, "head size %d is not one the attention kernels work on", head_dim);
    std::vector<int32_t> h((size_t)layers, kv_heads), d((size_t)layers, head_dim);
    return kv_create_keys(ctx, layers, h.data(), d.data(), type == TSB_F32 ? 4 : 2, page_tokens, num_pages, max_seqs, max_pages_per_seq, out);
}

int32_t tsb_window_attention(tsb_ctx* ctx, tsb_stream s, tsb_kv* keys, int32_t layer, const void* q, int64_t q_stride, void* out, int64_t out_stride,
                             const tsb_row_desc* rows_dev, const int32_t* group_rows, int32_t n_groups, int32_t n_q_heads, float scale, float cap,
                             const float* r1, const float* r2, const float* gate, int32_t window, int32_t max_len, void* scratch) {
    if (!ctx || !keys) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, !keys->key_layers.empty() && layer >= 0 && layer < (int)keys->key_layers.size(), "a key-only cache and one of its layers expected");
    TSB_REQUIRE(ctx, q && out && rows_dev && group_rows && n_groups > 0 && scratch && (r1 == nullptr) == (r2 == nullptr) && window >= 0, "bad arguments");
    const KeyView& kv = keys->key_layers[layer];
    TSB_REQUIRE(ctx, n_q_heads > 0 && n_q_heads % kv.kv_heads == 0 && wattn_supported(kv.head_dim, n_q_heads / kv.kv_heads, kv.elem_bytes == 4),
                "query heads must be a multiple of the key heads, at most %d per key head", WATTN_LARGE_Q);
    TSB_REQUIRE(ctx, (uintptr_t)q % 32 == 0 && (uintptr_t)out % 32 == 0 && q_stride % 16 == 0 && out_stride % 16 == 0 &&
                         q_stride >= (int64_t)n_q_heads * kv.head_dim && out_stride >= (int64_t)n_q_heads * kv.head_dim,
                "q and out rows hold every head and start on 32-byte boundaries (strides a multiple of 16)");
    cudaStream_t st = (cudaStream_t)s;
    DeviceGuard g(ctx);
    WindowAttn a;
    a.keys = kv, a.q = q, a.q_stride = q_stride, a.out = out, a.out_stride = out_stride, a.gate = gate, a.rows = rows_dev;
    a.n_q_heads = n_q_heads, a.scale = scale, a.cap = cap, a.r1 = r1, a.r2 = r2, a.window = window;
    AttnBatch b;
    b.max_len = max_len;
    bool uniform = true;
    for (int i = 0; i < n_groups; i++) {
        TSB_REQUIRE(ctx, group_rows[i] > 0, "every stream of the batch has rows");
        b.rows += group_rows[i];
        uniform &= group_rows[i] == group_rows[0];
    }
    if (uniform) {
        b.rows_per_seq = group_rows[0];
        TSB_CUDA(ctx, launch_window_attn(ctx, st, kv.elem_bytes == 4, a, b, scratch));
        return TSB_OK;
    }
    const int grp = n_q_heads / kv.kv_heads, rpt = wattn_rows_per_tile(kv.head_dim, grp);
    std::vector<AttnTile> small, large;
    for (int i = 0, r = 0; i < n_groups; r += group_rows[i], i++) {
        if (group_rows[i] * grp <= WATTN_SMALL_Q) {
            small.push_back({r, group_rows[i]});
            b.small_queries = std::max(b.small_queries, group_rows[i] * grp);
        } else {
            for (int k = 0; k < group_rows[i]; k += rpt) large.push_back({r + k, std::min(rpt, group_rows[i] - k)});
        }
    }
    b.n_small = (int)small.size(), b.n_large = (int)large.size();
    small.insert(small.end(), large.begin(), large.end());
    AttnTile* dev = nullptr;
    TSB_CUDA(ctx, cudaMallocAsync((void**)&dev, small.size() * sizeof(AttnTile), st));
    cudaError_t e = cudaMemcpyAsync(dev, small.data(), small.size() * sizeof(AttnTile), cudaMemcpyHostToDevice, st);
    b.small = dev, b.large = dev + b.n_small;
    if (e == cudaSuccess) e = launch_window_attn(ctx, st, kv.elem_bytes == 4, a, b, scratch);
    cudaError_t e2 = cudaFreeAsync(dev, st);
    TSB_CUDA(ctx, e);
    TSB_CUDA(ctx, e2);
    return TSB_OK;
}

}  // extern "C"
