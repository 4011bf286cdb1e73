// The plain-weight decoder family (tsb_model_create_plain): models, session buffers, forward pass.
//
// A layer in parallel form is four launches, plus the embedding before the first and norm + head after the last:
//   norm + token shift           f32 residual stream -> the mixer's input and the feed-forward's input
//   input matmul                 one packed matrix over queries | keys | head gates | gate-up pairs; its epilogue stores the
//                                queries, writes the keys into their cache slots, keeps the gates in f32 and leaves
//                                act(gate) * up beside the attention output
//   window attention             over the cache, gate applied where a head's output is finished
//   output matmul                [W_o | W_down] over [heads | feed-forward]: the two sublayers of a parallel layer add up
//                                inside one product, whose epilogue adds it to the stream
// In post-norm form the sublayers follow each other, each ending in an output matmul that adds to the scaled stream and a norm
// that rewrites the stream (f32) and its copy in the compute type.  Mixers of that form:
//   keys and values              input matmul over queries | keys | values (values go straight to the cache); norm per head of queries
//                                and keys, which writes the cache; attention
//   latent                       input matmul over queries | latent | value gates | rotated pairs, whose epilogue rotates queries
//                                and the shared key part in f32 and stores the latter in the cache; norm of the latent into the cache; then
//                                short portions: absorb (queries to the latent's space), attention over latent rows, lift (sums of
//                                latents to gated values); long portions: expansion of the stream's latents to keys and values, attention
// In output-norm form a sublayer reads the stream through a short convolution, and its output is normed and added by one kernel that also
// makes the next sublayer's input (launch_sublayer_end); the stream goes back and forth between two buffers.  Mixers: attention over keys
// and values, a recurrence (recurrence.cuh), or both side by side - one input matmul, one output matmul over [heads | recurrence].
// In pre-norm form a norm makes each sublayer's input, and its output matmul adds to the stream (f32).  Attention over keys and values there turns
// queries, keys and - if the layer says so - values with their positions in the kernel that norms them: coordinates of a pair are packed side by side
// (rows of W_q, W_k, W_v, columns of W_o), whichever layout the model stores.  Blocks before a window get their means behind it.
// Routed feed-forwards: router matmul, choice and lists, a grouped product each for gate-up pairs and down.
#include <algorithm>
#include <cstring>
#include <functional>
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
    uint64_t want = 1ull << TSB_P_EMBED | 1ull << TSB_P_HEAD | 1ull << TSB_P_FINAL_NORM;
    if (m->cfg.positions > 0) want |= 1ull << TSB_P_POSITIONS;
    TSB_REQUIRE(ctx, (m->set & want) == want, "embedding, head or final norm missing");
    for (size_t i = 0; i < m->layers.size(); i++) {
        const PlainLayer& l = m->layers[i];
        uint64_t w = 1ull << TSB_P_NORM;
        auto need = [&](bool on, std::initializer_list<int> ids) {
            for (int id : ids)
                if (on) w |= 1ull << id;
        };
        const int rec = l.cfg.recurrence;
        need(l.mixer != MIX_NONE, {TSB_P_Q, TSB_P_O});
        need(l.mixer == MIX_LATENT, {TSB_P_UK, TSB_P_UV});
        need(l.mixer == MIX_LATENT && l.source == (int)i, {TSB_P_DKV, TSB_P_DKV_NORM});
        need(l.mixer == MIX_KEYS || l.mixer == MIX_KV, {TSB_P_K});
        need(l.mixer == MIX_KV, {TSB_P_V});
        need(l.cfg.qk_norm, {TSB_P_Q_NORM, TSB_P_K_NORM});
        need(l.cfg.qkv_bias, {TSB_P_Q_BIAS, TSB_P_K_BIAS, TSB_P_V_BIAS});
        need(l.cfg.sink == TSB_SINK_TENSOR, {TSB_P_SINK});
        need(l.cfg.value_gate, {TSB_P_VALUE_GATE});
        need(l.cfg.token_shift, {TSB_P_SHIFT});
        need(l.cfg.head_gate, {TSB_P_HEAD_GATE});
        need(l.cfg.log_bias, {TSB_P_R1, TSB_P_R2});
        need(rec, {TSB_P_REC_O});
        need(rec && rec != TSB_REC_MINGRU, {TSB_P_REC_NORM});
        need(rec == TSB_REC_MINGRU, {TSB_P_REC_F, TSB_P_REC_F_BIAS, TSB_P_REC_I, TSB_P_REC_I_BIAS, TSB_P_REC_GATE});
        need(rec == TSB_REC_FORGET || rec == TSB_REC_MLSTM, {TSB_P_REC_Q, TSB_P_REC_V, TSB_P_REC_F, TSB_P_REC_F_BIAS});
        need(rec == TSB_REC_FORGET, {TSB_P_REC_LOWER});
        need(rec == TSB_REC_MLSTM, {TSB_P_REC_K, TSB_P_REC_GATE, TSB_P_REC_I, TSB_P_REC_I_BIAS});
        need(rec == TSB_REC_SSD, {TSB_P_REC_IN, TSB_P_REC_CONV, TSB_P_REC_CONV_BIAS, TSB_P_REC_DT_BIAS, TSB_P_REC_A_LOG, TSB_P_REC_D});
        need(m->cfg.conv_taps > 0, {TSB_P_CONV1});
        need(m->cfg.conv_taps > 0 && l.cfg.ffn > 0, {TSB_P_CONV2});
        need(l.cfg.ffn > 0, {TSB_P_FF_UP, TSB_P_FF_DOWN});
        need(l.cfg.ffn > 0 && !l.cfg.ff_plain, {TSB_P_FF_GATE});
        need(l.cfg.ffn > 0 && l.post_norm, {TSB_P_NORM2});
        need(l.cfg.experts > 0, {TSB_P_ROUTER, TSB_P_CORRECTION});
        TSB_REQUIRE(ctx, (l.set & w) == w, "layer %zu is missing a tensor (have %llx, need %llx)", i, (unsigned long long)l.set, (unsigned long long)w);
    }
    return TSB_OK;
}

void free_layer(tsb_ctx* ctx, PlainLayer& l) {
    if (!l.owned) return;
    for (void** p : l.buffers())
        if (*p) tsb_free(ctx, *p);
}

// layers that use the tensors of layer `from` get its pointers
void mirror_layer(PlainModel* m, int from) {
    for (int i = 0; i < m->cfg.n_layers; i++) {
        PlainLayer& l = m->layers[i];
        if (l.tied != from) continue;
        const tsb_plain_layer cfg = l.cfg;
        const int source = l.source;
        l = m->layers[from];
        l.cfg = cfg, l.source = source, l.tied = from, l.owned = false;
    }
}

void plain_free(tsb_model* tm) {
    PlainModel* m = tm->plain;
    if (!m) return;
    tsb_ctx* ctx = tm->ctx;
    for (PlainLayer& l : m->layers) free_layer(ctx, l);
    for (PlainRotation& r : m->rotations)
        if (r.freq) tsb_free(ctx, r.freq);
    if (m->owned)
        for (void* p : {m->head.data, m->embed, m->positions, (void*)m->final_gain})
            if (p) tsb_free(ctx, p);
    delete m;
    tm->plain = nullptr;
}

// rows of a recurrence in the input matrix: vectors in the compute type, gates in f32
int64_t rec_typed_rows(const tsb_plain_layer& c) {
    const int64_t h = c.rec_heads, D = c.rec_dim, E = c.rec_vdim;
    return c.recurrence == TSB_REC_MINGRU ? E : c.recurrence == TSB_REC_FORGET ? h * (D + E) : c.recurrence == TSB_REC_MLSTM ? 2 * h * (D + E) : c.recurrence == TSB_REC_SSD ? 2 * h * E + 2 * c.rec_groups * D : 0;
}
int64_t rec_gate_rows(const tsb_plain_layer& c) {
    const int64_t h = c.rec_heads;
    return c.recurrence == TSB_REC_MINGRU ? 2 * (int64_t)c.rec_vdim : c.recurrence == TSB_REC_FORGET ? h * c.rec_dim : c.recurrence == TSB_REC_MLSTM ? 2 * h : c.recurrence == TSB_REC_SSD ? h : 0;
}
int64_t rec_conv_channels(const tsb_plain_layer& c) { return c.recurrence == TSB_REC_SSD ? (int64_t)c.rec_heads * c.rec_vdim + 2 * (int64_t)c.rec_groups * c.rec_dim : 0; }
// numbers of a layer's matrices that a pass over one row reads
int64_t layer_numbers(const PlainLayer& l, int64_t d) {
    const tsb_plain_layer& c = l.cfg;
    const int64_t H = c.n_q_heads, G = c.n_kv_heads, D = c.head_dim, E = l.mixer == MIX_KEYS ? D : c.value_dim;
    int64_t n = d * (H * E + (c.head_gate ? H : 0) + (c.value_gate ? H * E : 0));
    n += c.experts > 0 ? d * (c.experts + 3 * (int64_t)c.ffn * c.expert_top) : d * (c.ff_plain ? 2 : 3) * (int64_t)c.ffn;
    n += d * (rec_typed_rows(c) + rec_gate_rows(c) + (c.recurrence ? (int64_t)c.rec_heads * c.rec_vdim : 0));
    if (l.mixer == MIX_LATENT) {
        n += d * H * (D + c.rot_dim) + (int64_t)c.kv_rank * H * (D + E);
        if (c.kv_source == 0) n += d * (c.kv_rank + c.rot_dim);
    } else if (l.mixer != MIX_NONE) {
        n += d * (H * D + G * D + (l.mixer == MIX_KV ? G * E : 0));
    }
    return n;
}
// bytes a pass reads of the matrices (the embedding is read by rows and not counted)
int64_t plain_weight_bytes(const tsb_model* tm) {
    const PlainModel* m = tm->plain;
    int64_t n = (int64_t)m->cfg.vocab * m->cfg.d_model;
    for (const PlainLayer& l : m->layers) n += layer_numbers(l, m->cfg.d_model);
    return n * m->elem;
}

int32_t plain_share(tsb_model* dt, int32_t dst_layer, const tsb_model* st, int32_t src_layer) {
    tsb_ctx* ctx = dt->ctx;
    PlainModel* d = dt->plain;
    const PlainModel* s = st->plain;
    TSB_REQUIRE(ctx, d->cfg.d_model == s->cfg.d_model && d->cfg.vocab == s->cfg.vocab && d->f32 == s->f32 && d->cfg.post_norm == s->cfg.post_norm &&
                         d->cfg.output_norm == s->cfg.output_norm && d->cfg.pre_norm == s->cfg.pre_norm && d->cfg.conv_taps == s->cfg.conv_taps && d->cfg.positions == s->cfg.positions,
                "models differ in width, vocabulary, type or form");
    if (dst_layer < 0) {
        if (d->owned)
            for (void* p : {d->head.data, d->embed, d->positions, (void*)d->final_gain})
                if (p) tsb_free(ctx, p);
        d->head = s->head, d->embed = s->embed, d->positions = s->positions, d->final_gain = s->final_gain, d->set = s->set, d->owned = false;
        return TSB_OK;
    }
    TSB_REQUIRE(ctx, dst_layer < d->cfg.n_layers && src_layer >= 0 && src_layer < s->cfg.n_layers, "layer out of range");
    PlainLayer& l = d->layers[dst_layer];
    TSB_REQUIRE(ctx, l.tied < 0, "layer %d uses the tensors of layer %d", dst_layer, l.tied);
    const tsb_plain_layer own = l.cfg;
    tsb_plain_layer theirs = s->layers[src_layer].cfg;
    theirs.weights_of = 0;
    TSB_REQUIRE(ctx, memcmp(&own, &theirs, sizeof own) == 0, "layer shapes differ");
    free_layer(ctx, l);
    const int rotation = l.rotation, value_rotation = l.value_rotation, source = l.source;
    l = s->layers[src_layer];
    l.cfg = own, l.rotation = rotation, l.value_rotation = value_rotation, l.source = source;
    l.tied = -1, l.owned = false;
    mirror_layer(d, dst_layer);
    return TSB_OK;
}

void plain_runtime_free(ModelRt& rt) {
    delete rt.plain;  // the device buffers belong to the session
    rt.plain = nullptr;
}

constexpr int CHUNK_MIN_ROWS = 32;  // rows of a portion from which on its recurrences go chunk by chunk
// Rings of the convolutions and states of the recurrences.  A cursor may go back by max_rows rows after a pass of as many, so the states of
// max_rows + 1 positions are kept, and the convolutions' inputs as far back as the oldest of them looks.
int32_t states_init(tsb_session* s, const PlainModel* m, const SessionShape& shape, StreamStates& st) {
    tsb_ctx* ctx = s->ctx;
    auto zero = [&](size_t bytes, void** q) -> int32_t {
        if (bytes == 0) return TSB_OK;
        if (int32_t rc = dev_alloc(ctx, s->owned, bytes, q)) return rc;
        TSB_CUDA(ctx, cudaMemset(*q, 0, bytes));
        return TSB_OK;
    };
    bool any = m->cfg.conv_taps > 1;
    st.keep = std::max(0, m->cfg.conv_taps - 1);
    for (const PlainLayer& l : m->layers)
        if (l.cfg.recurrence) any = true, st.keep = std::max(st.keep, l.cfg.rec_taps - 1);
    if (!any) return TSB_OK;
    for (st.ring = 2; st.ring < shape.max_rows + 1;) st.ring *= 2;
    for (st.row_ring = 2; st.row_ring < st.ring + st.keep;) st.row_ring *= 2;
    std::vector<RowRing> rings;
    size_t scratch = 0, sums = 0;
    int32_t rc = TSB_OK;
    auto ring = [&](std::vector<RowRing>& list, int64_t width, int taps) {
        RowRing r;
        r.width = (int)width, r.ring_rows = st.row_ring, r.keep = std::max(0, taps - 1), r.n_streams = shape.n_streams;
        if (width > 0 && r.keep > 0 && rc == TSB_OK) {
            const size_t row = (size_t)shape.n_streams * width * 4;
            rc = zero(row * r.ring_rows, (void**)&r.ring);
            if (rc == TSB_OK) rc = zero(row * r.keep, (void**)&r.before);
            rings.push_back(r);
        }
        list.push_back(r);
    };
    for (const PlainLayer& l : m->layers) {
        const tsb_plain_layer& c = l.cfg;
        ring(st.conv1, m->cfg.d_model, m->cfg.conv_taps);
        ring(st.conv2, c.ffn > 0 ? m->cfg.d_model : 0, m->cfg.conv_taps);
        ring(st.rec, rec_conv_channels(c), c.rec_taps);
        RecurrentState r;
        r.ring = st.ring, r.n_streams = shape.n_streams;
        const size_t heads = (size_t)shape.n_streams * st.ring * c.rec_heads;
        if (c.recurrence && rc == TSB_OK) rc = zero(heads * c.rec_dim * recurrence_v_pitch(c.rec_vdim) * 4, (void**)&r.s);
        const size_t copies = heads * recurrence_copies(c.rec_vdim);
        if (c.recurrence == TSB_REC_MLSTM && rc == TSB_OK) rc = zero(copies * c.rec_dim * 4, (void**)&r.norm);
        if (c.recurrence == TSB_REC_MLSTM && rc == TSB_OK) rc = zero(copies * 8, (void**)&r.top);
        if (c.recurrence == TSB_REC_MINGRU) sums = std::max(sums, (size_t)(shape.pass_rows / SCAN_CHUNK + shape.n_streams) * c.rec_vdim * sizeof(float2));
        else if (c.recurrence && !m->f32)
            scratch = std::max(scratch, recurrence_scratch_bytes(c.recurrence, c.rec_heads, c.rec_dim, c.rec_vdim, shape.pass_rows / REC_CHUNK + shape.n_streams));
        st.states.push_back(r);
    }
    if (rc == TSB_OK && shape.pass_rows >= CHUNK_MIN_ROWS) rc = zero(scratch, &st.chunk_scratch);
    if (rc == TSB_OK && shape.pass_rows > SCAN_CHUNK) rc = zero(sums, (void**)&st.scan_sums);
    if (rc) return rc;
    st.n_rings = (int)rings.size();
    if (st.n_rings == 0) return TSB_OK;
    if ((rc = zero(rings.size() * sizeof(RowRing), (void**)&st.rings_dev))) return rc;
    TSB_CUDA(ctx, cudaMemcpy(st.rings_dev, rings.data(), rings.size() * sizeof(RowRing), cudaMemcpyHostToDevice));
    return TSB_OK;
}

constexpr int EXPAND_MIN_ROWS = 64;                 // rows of a portion from which on its latents are expanded
constexpr size_t EXPAND_MAX_BYTES = 2ull << 30;

int32_t plain_runtime_init(tsb_session* s, ModelRt& rt, const tsb_model* tm, const SessionShape& shape, bool is_draft) {
    (void)is_draft;
    tsb_ctx* ctx = s->ctx;
    const PlainModel* m = tm->plain;
    rt.model = tm;
    std::vector<KeyLayerShape> shapes;
    for (const PlainLayer& l : m->layers) {
        if (l.mixer == MIX_LATENT) shapes.push_back({1, l.key_dim, 0, l.source});
        else if (l.mixer == MIX_NONE) shapes.push_back({0, 0, 0, (int)shapes.size()});
        else shapes.push_back({l.cfg.n_kv_heads, l.head_pad, l.mixer == MIX_KV ? l.head_pad : 0, (int)shapes.size(), l.cfg.pool});
    }
    int32_t rc = kv_create_keys(ctx, m->cfg.n_layers, shapes.data(), m->elem, shape.page_tokens, shape.num_pages, shape.n_streams, shape.pages_per_seq, &rt.kv);
    if (rc) return rc;
    PlainRt* p = rt.plain = new (std::nothrow) PlainRt();
    if (!p) return TSB_ERR_OOM;
    // matmul operands are read in whole token tiles
    p->rows = (int)plain_pad(std::max(shape.pass_rows, 32), 32);
    p->in_stride = m->d_pad;
    int64_t wide = 0, latent = 0, experts = 0, top = 0, expert_ffn = 0;
    for (const PlainLayer& l : m->layers) {
        const int64_t H = l.cfg.n_q_heads, inner = (int64_t)l.cfg.rec_heads * l.cfg.rec_vdim;
        p->rec_stride = std::max<int64_t>(p->rec_stride, plain_pad(rec_typed_rows(l.cfg), 16));
        p->rec_mixed_stride = std::max<int64_t>(p->rec_mixed_stride, plain_pad(rec_conv_channels(l.cfg), 16));
        if (l.cfg.recurrence && l.cfg.recurrence != TSB_REC_MINGRU) p->rec_out_stride = std::max<int64_t>(p->rec_out_stride, plain_pad(inner, 4));
        const int64_t heads = l.cfg.qk_norm ? plain_pad((H + l.cfg.n_kv_heads) * l.cfg.head_dim + (l.cfg.value_rot ? l.cfg.n_kv_heads * l.cfg.value_dim : 0), 4) : 0;
        p->raw_stride = std::max<int64_t>(p->raw_stride, heads);
        if (l.cfg.recurrence) p->raw_rec = std::max<int64_t>(p->raw_rec, heads);
        if (l.cfg.experts > 0)
            experts = std::max<int64_t>(experts, l.cfg.experts), top = std::max<int64_t>(top, l.cfg.expert_top), expert_ffn = std::max<int64_t>(expert_ffn, l.ffn_pad);
        p->q_stride = std::max<int64_t>(p->q_stride, plain_pad(H * l.head_pad, 16));
        p->cat_stride = std::max<int64_t>(p->cat_stride, l.out.cols);
        p->gate_stride = std::max(p->gate_stride, l.cfg.n_q_heads);
        if (l.post_norm && l.cfg.experts == 0) p->act_stride = std::max<int64_t>(p->act_stride, l.ffn_pad);
        if (l.cfg.value_gate) p->value_gate_stride = std::max<int64_t>(p->value_gate_stride, plain_pad(H * l.value_pad, 16));
        if (l.mixer != MIX_LATENT) continue;
        p->raw_stride = std::max<int64_t>(p->raw_stride, plain_pad(l.cfg.kv_rank, 4));
        p->absorbed_stride = std::max<int64_t>(p->absorbed_stride, H * l.key_dim);
        p->sums_stride = std::max<int64_t>(p->sums_stride, H * l.rank_pad);
        if (l.expands) wide = std::max<int64_t>(wide, H * (l.head_pad + l.value_pad)), latent = std::max<int64_t>(latent, l.key_dim);
    }
    for (const PlainLayer& l : m->layers)
        if (l.cfg.recurrence) p->raw_stride = std::max<int64_t>(p->raw_stride, plain_pad(p->raw_rec + rec_gate_rows(l.cfg), 4));
    p->fin_rows = (int)plain_pad(std::max(std::max(shape.n_streams * shape.max_rows, std::min(shape.pass_rows, 256)), 32), 32);
    auto A = [&](size_t bytes, void** q) {
        if (bytes == 0) return (int32_t)TSB_OK;
        int32_t r = dev_alloc(ctx, s->owned, bytes, q);
        if (r == TSB_OK && cudaMemset(*q, 0, bytes) != cudaSuccess) r = tsb_fail(ctx, TSB_ERR_CUDA, "clearing a work buffer failed");
        return r;
    };
    const size_t R = p->rows, e = m->elem;
    if ((rc = A(R * m->cfg.d_model * 4, (void**)&p->x)) || (rc = A(R * p->in_stride * e, &p->mix)) ||
        (rc = A(m->sequential() ? 0 : R * p->in_stride * e, &p->h)) || (rc = A(R * p->q_stride * e, &p->q)) || (rc = A(R * p->cat_stride * e, &p->cat)) ||
        (rc = A(R * p->gate_stride * 4, (void**)&p->gate)) || (rc = A((size_t)p->fin_rows * p->in_stride * e, &p->fin)) ||
        (rc = A(plain_gemm_workspace_bytes(ctx), &p->gemm_ws)) || (rc = A(wattn_scratch_bytes(ctx), &p->attn_ws)) ||
        (rc = A(R * p->act_stride * e, &p->act)) || (rc = A(R * p->raw_stride * 4, (void**)&p->raw)) || (rc = A(R * p->absorbed_stride * e, &p->absorbed)) ||
        (rc = A(R * p->sums_stride * e, &p->sums)) || (rc = A(R * p->value_gate_stride * e, &p->value_gate)))
        return rc;
    if (m->cfg.output_norm) {
        const size_t slots = plain_pad(R * top, 32) + 256;  // token tiles of a product may reach behind the last slot
        p->expert_rows = top > 0 ? (int)slots : 0;
        if ((rc = A(R * m->cfg.d_model * 4, (void**)&p->x2)) || (rc = A(R * m->cfg.d_model * 4, (void**)&p->y))) return rc;
        if (top > 0) {
            ExpertLists& x = p->lists;
            const size_t ints = R * top * sizeof(int32_t);
            if ((rc = A(R * experts * 4, (void**)&p->router_logits)) || (rc = A(slots * p->in_stride * e, &p->expert_in)) ||
                (rc = A(slots * expert_ffn * e, &p->expert_act)) || (rc = A(slots * m->cfg.d_model * e, &p->expert_out)) || (rc = A(ints, (void**)&x.ids)) ||
                (rc = A(ints, (void**)&x.weight)) || (rc = A(ints, (void**)&x.slot_of)) || (rc = A(ints, (void**)&x.token_of)) ||
                (rc = A((experts + 1) * sizeof(int32_t), (void**)&x.first)) || (rc = A((experts + R * top / 8 + 1) * sizeof(ExpertChunk), (void**)&x.chunks)) ||
                (rc = A(sizeof(int32_t), (void**)&x.n_chunks)))
                return rc;
        }
    }
    if (m->cfg.output_norm || m->cfg.pre_norm) {
        if ((rc = A(R * p->rec_stride * e, &p->rec)) || (rc = A(R * p->rec_mixed_stride * e, &p->rec_mixed)) || (rc = A(R * p->rec_out_stride * 4, (void**)&p->rec_out))) return rc;
        if ((rc = states_init(s, m, shape, p->states))) return rc;
        if (p->states.ring > 0) rt.kv->state_ring = p->states.ring + 1;
    }
    for (const PlainRotation& r : m->rotations) {
        float2* t = nullptr;
        if ((rc = A(R * (r.dims / 2) * sizeof(float2), (void**)&t))) return rc;
        p->rotary.push_back(t);
    }
    if (wide > 0 && shape.pass_rows >= EXPAND_MIN_ROWS) {
        ExpandRt& x = p->expand;
        const int64_t tokens = (int64_t)shape.num_pages * shape.page_tokens;
        const int64_t room = (int64_t)(EXPAND_MAX_BYTES / ((size_t)(wide + latent) * e));
        x.pages = (int)std::min<int64_t>(tokens / EXPAND_PAGE + shape.n_streams, room / EXPAND_PAGE);
        x.max_seqs = shape.n_streams;
        x.pages_per_seq = (int)(((int64_t)shape.pages_per_seq * shape.page_tokens + EXPAND_PAGE - 1) / EXPAND_PAGE);
        if ((rc = A((size_t)x.pages * EXPAND_PAGE * wide * e, &x.wide)) || (rc = A((size_t)x.pages * EXPAND_PAGE * latent * e, &x.latents)) ||
            (rc = A((size_t)x.max_seqs * x.pages_per_seq * sizeof(int32_t), (void**)&x.table)))
            return rc;
    }
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

// ------------------------------------------------------------------ packed rows of a layer's input matrix
struct InRows {
    int64_t q = 0, k = 0, v = 0, head_gate = 0, value_gate = 0;  // first rows; latent layers: k is the latent
    int64_t rec = 0, rec_gate = 0;                               // of the recurrence's vectors and gates
    int64_t segments = 0;                                        // end of the rows with destinations of their own
    int64_t pairs = 0, n_pairs = 0;                              // interleaved pairs behind them (gate and up, or rotated coordinates)
    int64_t rows = 0;
};
InRows in_rows(const PlainLayer& l) {
    const tsb_plain_layer& c = l.cfg;
    const int64_t H = c.n_q_heads, G = c.n_kv_heads, E = c.value_dim;
    const bool own = c.kv_source == 0;
    InRows r;
    int64_t at = l.mixer == MIX_NONE ? 0 : l.mixer == MIX_KEYS ? l.q_rows : H * c.head_dim;
    r.k = at;
    at += l.mixer == MIX_NONE ? 0 : l.mixer == MIX_KEYS ? l.k_rows : l.mixer == MIX_KV ? G * c.head_dim : own ? c.kv_rank : 0;
    r.v = at;
    if (l.mixer == MIX_KV) at += G * E;
    r.head_gate = at;
    if (c.head_gate) at += H;
    r.value_gate = at;
    if (c.value_gate) at += H * E;
    r.rec = at;
    at += rec_typed_rows(c);
    r.rec_gate = at;
    at += rec_gate_rows(c);
    r.segments = at;
    r.pairs = plain_pad(at, PLAIN_ROW_PAD);
    if (l.mixer == MIX_LATENT) r.n_pairs = (H + (own ? 1 : 0)) * (c.rot_dim / 2);
    else if (!l.post_norm) r.n_pairs = l.ffn_pad;
    r.rows = r.pairs + plain_pad(2 * plain_pad(r.n_pairs, 8), PLAIN_ROW_PAD);
    return r;
}

// ------------------------------------------------------------------ forward pass
// The query tiles of a ragged pass for one geometry, and which streams of the pass they are made of.
enum TileSet { TILES_ALL = 0, TILES_LATENT, TILES_LATENT_SHORT, TILES_WIDE };
struct TileLists {
    int set, group, rows_per_tile;
    AttnBatch batch;
};
// What a pass knows about its portions before the first launch.
struct PassPlan {
    std::vector<TileLists> lists;
    int max_len = 0, longest = 0, longest_short = 0, rows_short = 0;
    // portions whose latents are expanded, and the rows that hold all the others
    std::vector<ExpandStream> expanded;
    std::vector<bool> is_expanded;
    const ExpandStream* expanded_dev = nullptr;
    int expanded_pages = 0, expanded_len = 0, short_first = 0, short_rows = 0;
    // output-norm form and recurrences: runs of rows for the row operators; portions whose recurrences go row by row, and chunk by chunk where there is a kernel
    RowTiles runs, by_row, portions;  // portions: all of them
    RowTiles scan_chunks;             // those that are not in by_row, in chunks for element-wise recurrences
    bool several_chunks = false;      // of one portion
    RecurrenceChunks by_chunk;
    bool use_before = false;

    const AttnBatch* find(int set, int group, int rows_per_tile) const {
        for (const TileLists& t : lists)
            if (t.set == set && t.group == group && t.rows_per_tile == rows_per_tile) return &t.batch;
        return nullptr;
    }
};

LatentTiling latent_tiling(const tsb_ctx* ctx, const PassPlan& plan, const Pass& p, const PlainLayer& l) {
    const bool all = p.rows_per_seq > 0 || !l.expands;
    return latent_attn_tiling(ctx, l.cfg.n_q_heads, all ? plan.longest : plan.longest_short, all ? p.rows : plan.rows_short, plan.max_len);
}

int32_t plan_states(tsb_session* s, const PlainModel* m, const ModelRt& rt, const Pass& p, PassPlan& plan) {
    const StreamStates& states = rt.plain->states;
    plan.use_before = states.n_rings > 0 && plan.longest + states.keep > states.row_ring;
    const int per = sublayer_rows_per_tile(s->ctx, p.rows);
    if (p.rows_per_seq > 0) {
        plan.runs = RowTiles::uniform(p.rows, p.rows_per_seq, per);
        plan.by_row = plan.portions = RowTiles::uniform(p.rows, p.rows_per_seq, p.rows_per_seq);
        return TSB_OK;
    }
    std::vector<AttnTile> runs, by_row, scan_chunks, portions, chunks;
    std::vector<ChunkPortion> by_chunk;
    for (int i = 0; i < p.n_groups; i++) {
        const RowGroup& g = p.groups[i];
        for (int r = 0; r < g.n_rows; r += per) runs.push_back({g.first_row + r, std::min(per, g.n_rows - r)});
        const bool long_portion = !m->f32 && g.n_rows >= CHUNK_MIN_ROWS;
        portions.push_back({g.first_row, g.n_rows});
        if (!long_portion) {
            by_row.push_back({g.first_row, g.n_rows});
            continue;
        }
        for (int r = 0; r < g.n_rows; r += SCAN_CHUNK) scan_chunks.push_back({g.first_row + r, std::min(SCAN_CHUNK, g.n_rows - r)});
        plan.several_chunks |= g.n_rows > SCAN_CHUNK;
        by_chunk.push_back({g.first_row, g.n_rows, (int)chunks.size()});
        for (int r = 0; r < g.n_rows; r += REC_CHUNK) chunks.push_back({g.first_row + r, std::min(REC_CHUNK, g.n_rows - r)});
        rt.kv->state_lo[g.seq] = g.base + g.n_rows - 1;  // the states in between are not kept
    }
    auto stage = [&](const std::vector<AttnTile>& list, RowTiles& out) -> int32_t {
        if (list.empty()) {
            out.n = 0;
            return TSB_OK;
        }
        const int32_t* dev = nullptr;
        if (int32_t rc = session_stage_ints(s, reinterpret_cast<const int32_t*>(list.data()), (int)list.size() * 2, &dev)) return rc;
        out = RowTiles::list(reinterpret_cast<const AttnTile*>(dev), (int)list.size());
        for (const AttnTile& t : list) out.longest = std::max(out.longest, t.n_rows);
        return TSB_OK;
    };
    int32_t rc = stage(runs, plan.runs);
    if (rc == TSB_OK) rc = stage(by_row, plan.by_row);
    if (rc == TSB_OK) rc = stage(portions, plan.portions);
    if (rc == TSB_OK) rc = stage(scan_chunks, plan.scan_chunks);
    if (rc == TSB_OK) rc = stage(chunks, plan.by_chunk.chunks);
    if (rc || by_chunk.empty()) return rc;
    const int32_t* dev = nullptr;
    if ((rc = session_stage_ints(s, reinterpret_cast<const int32_t*>(by_chunk.data()), (int)by_chunk.size() * 3, &dev))) return rc;
    plan.by_chunk.portions = reinterpret_cast<const ChunkPortion*>(dev), plan.by_chunk.n_portions = (int)by_chunk.size();
    plan.by_chunk.scratch = states.chunk_scratch;
    return TSB_OK;
}

int32_t plan_pass(tsb_session* s, const PlainModel* m, const ModelRt& rt, const Pass& p, PassPlan& plan) {
    const PlainRt* b = rt.plain;
    plan.max_len = (p.max_len + 511) / 512 * 512;  // the split plan changes only every 512 positions (graph reuse)
    plan.longest = p.rows_per_seq;
    plan.short_rows = p.rows;
    const bool states = m->cfg.output_norm || b->states.ring > 0;
    if (p.rows_per_seq > 0) return states ? plan_states(s, m, rt, p, plan) : TSB_OK;
    plan.is_expanded.assign(p.n_groups, false);
    int first_short = p.rows, end_short = 0;
    for (int i = 0; i < p.n_groups; i++) {
        const RowGroup& g = p.groups[i];
        plan.longest = std::max(plan.longest, g.n_rows);
        const int len = (int)g.base + g.n_rows, pages = (len + EXPAND_PAGE - 1) / EXPAND_PAGE;
        if (g.n_rows >= EXPAND_MIN_ROWS && plan.expanded_pages + pages <= b->expand.pages) {
            plan.is_expanded[i] = true;
            plan.expanded.push_back({g.first_row, g.n_rows, plan.expanded_pages});
            plan.expanded_pages += pages, plan.expanded_len = std::max(plan.expanded_len, len);
        } else {
            first_short = std::min(first_short, g.first_row), end_short = std::max(end_short, g.first_row + g.n_rows);
            plan.longest_short = std::max(plan.longest_short, g.n_rows), plan.rows_short += g.n_rows;
        }
    }
    plan.short_first = first_short, plan.short_rows = std::max(0, end_short - first_short);
    if (!plan.expanded.empty()) {
        const int32_t* dev = nullptr;
        if (int32_t rc = session_stage_ints(s, reinterpret_cast<const int32_t*>(plan.expanded.data()), (int)plan.expanded.size() * 3, &dev)) return rc;
        plan.expanded_dev = reinterpret_cast<const ExpandStream*>(dev);
    }
    if (states)
        if (int32_t rc = plan_states(s, m, rt, p, plan)) return rc;
    if (m->f32) return TSB_OK;  // the f32 kernel takes rows one by one
    auto add = [&](int set, int group, int rpt, int small_queries) -> int32_t {
        if (plan.find(set, group, rpt)) return TSB_OK;
        std::vector<AttnTile> small, large;
        TileLists t;
        t.set = set, t.group = group, t.rows_per_tile = rpt;
        for (int i = 0; i < p.n_groups; i++) {
            const RowGroup& g = p.groups[i];
            if ((set == TILES_LATENT_SHORT && plan.is_expanded[i]) || (set == TILES_WIDE && !plan.is_expanded[i])) continue;
            if (g.n_rows * group <= small_queries) {
                small.push_back({g.first_row, g.n_rows});
                t.batch.small_queries = std::max(t.batch.small_queries, g.n_rows * group);
            } else {
                for (int r = 0; r < g.n_rows; r += rpt) large.push_back({g.first_row + r, std::min(rpt, g.n_rows - r)});
            }
        }
        if (set == TILES_LATENT || set == TILES_LATENT_SHORT) small.swap(large);
        t.batch.n_small = (int)small.size(), t.batch.n_large = (int)large.size();
        small.insert(small.end(), large.begin(), large.end());
        const int32_t* dev = nullptr;
        if (int32_t rc = session_stage_ints(s, reinterpret_cast<const int32_t*>(small.data()), (int)small.size() * 2, &dev)) return rc;
        t.batch.small = reinterpret_cast<const AttnTile*>(dev), t.batch.large = t.batch.small + t.batch.n_small;
        t.batch.rows = p.rows, t.batch.max_len = plan.max_len;
        plan.lists.push_back(t);
        return TSB_OK;
    };
    for (const PlainLayer& l : m->layers) {
        int32_t rc = TSB_OK;
        if (l.mixer == MIX_NONE) continue;
        if (l.mixer != MIX_LATENT) {
            const int grp = l.cfg.n_q_heads / l.cfg.n_kv_heads;
            rc = add(TILES_ALL, grp, wattn_rows_per_tile(l.head_pad, grp, l.cfg.log_bias != 0), WATTN_SMALL_Q);
        } else {
            if (!l.expands || plan.longest_short > 0)
                rc = add(l.expands ? TILES_LATENT_SHORT : TILES_LATENT, l.cfg.n_q_heads, latent_tiling(s->ctx, plan, p, l).rows, 0);
            if (rc == TSB_OK && l.expands && !plan.expanded.empty()) rc = add(TILES_WIDE, 1, WATTN_WIDE_ROWS, 0);
        }
        if (rc) return rc;
    }
    return TSB_OK;
}

struct Forward {
    tsb_session* s;
    ModelRt& rt;
    const Pass& p;
    tsb_ctx* ctx;
    cudaStream_t st;
    const PlainModel* m;
    PlainRt* b;
    const PassPlan& plan;

    void* at(void* base, int64_t elements) const { return static_cast<uint8_t*>(base) + (size_t)elements * m->elem; }
    cudaError_t matmul(const PlainMat& w, const void* x, const void* x2, int64_t stride, const PlainEpi& epi) const {
        return launch_plain_gemm(ctx, st, m->f32, w, x, x2, stride, b->rows, p.rows, epi, b->gemm_ws);
    }

    // projections of a layer: x to the mixer's rows, x2 to the (gate, up) pairs of a parallel layer
    cudaError_t project(int L, const void* x, const void* x2) const {
        const PlainLayer& l = m->layers[L];
        const tsb_plain_layer& c = l.cfg;
        const InRows r = in_rows(l);
        PlainEpi e;
        e.kind = PLAIN_MIXER, e.keys = rt.kv->key_layers[L], e.rows = p.rows_dev, e.bias = l.in_bias;
        auto seg = [&](int64_t end, int kind, void* to, int64_t stride, int64_t per = 0x7fffffff, int64_t step = 0) {
            PlainSeg& g = e.seg[e.n_seg++];
            g.end = (int)end, g.kind = kind, g.p = to, g.stride = stride, g.per = (int)per, g.step = (int)step;
        };
        if (l.mixer == MIX_KEYS) {
            seg(r.k, PLAIN_SEG_TYPED, b->q, b->q_stride);
            seg(r.v, PLAIN_SEG_CACHE, nullptr, 0);
        } else if (l.mixer == MIX_KV) {
            if (c.qk_norm) {
                seg(c.value_rot ? r.head_gate : r.v, PLAIN_SEG_F32, b->raw, b->raw_stride);
            } else {
                seg(r.k, PLAIN_SEG_TYPED, b->q, b->q_stride, c.head_dim, l.head_pad);
                seg(r.v, PLAIN_SEG_CACHE, nullptr, 0, c.head_dim, e.keys.head_step);
            }
            if (!c.value_rot) seg(r.head_gate, PLAIN_SEG_CACHE, nullptr, e.keys.value_off, c.value_dim, e.keys.head_step);
        } else if (l.mixer == MIX_LATENT) {
            seg(r.k, PLAIN_SEG_TYPED, b->q, b->q_stride, c.head_dim, l.head_pad);
            if (r.v > r.k) seg(r.v, PLAIN_SEG_F32, b->raw, b->raw_stride);
            if (c.rot_dim > 0) {
                PlainRotate& t = e.rot;
                t.half = c.rot_dim / 2, t.n_heads = c.n_q_heads, t.table = b->rotary[l.rotation], t.key_off = c.kv_rank;
                t.q[0] = b->q, t.q_stride[0] = b->q_stride, t.q_step[0] = l.head_pad, t.q_off[0] = c.head_dim;
                t.q[1] = b->absorbed, t.q_stride[1] = b->absorbed_stride, t.q_step[1] = l.key_dim, t.q_off[1] = c.kv_rank;
            }
        }
        if (c.head_gate) seg(r.value_gate, PLAIN_SEG_F32, b->gate, c.n_q_heads);
        if (c.value_gate) seg(r.rec, PLAIN_SEG_TYPED, b->value_gate, b->value_gate_stride, c.value_dim, l.value_pad);
        if (c.recurrence) {
            seg(r.rec_gate, PLAIN_SEG_TYPED, b->rec, b->rec_stride);
            seg(r.segments, PLAIN_SEG_F32, b->raw + b->raw_rec, b->raw_stride);
        }
        if (r.n_pairs > 0) {
            e.pair_row0 = (int)r.pairs, e.n_pairs = (int)r.n_pairs, e.act = c.act;
            e.a = at(b->cat, l.o_cols), e.a_stride = l.out.cols;  // a rotation does not use them
        }
        return matmul(l.in, x, x2, b->in_stride, e);
    }

    cudaError_t head_norms(int L) const {
        const PlainLayer& l = m->layers[L];
        const tsb_plain_layer& c = l.cfg;
        HeadNorms h;
        h.raw = b->raw, h.raw_stride = b->raw_stride, h.eps = m->cfg.norm_eps, h.keys = rt.kv->key_layers[L], h.rows = p.rows_dev;
        if (l.mixer == MIX_LATENT) {
            h.n_k = 1, h.width = c.kv_rank, h.k_weight = l.c_norm;
        } else {
            h.n_q = c.n_q_heads, h.n_k = c.n_kv_heads, h.width = c.head_dim, h.q_weight = l.q_norm, h.k_weight = l.k_norm;
            h.temp_coef = c.q_temp_coef, h.temp_every = c.q_temp_every;
            h.q = b->q, h.q_stride = b->q_stride, h.q_step = h.q_width = l.head_pad;
            if (l.rotation >= 0) h.rot = b->rotary[l.rotation], h.rot_half = c.rot_dim / 2;
            if (c.pool > 0) h.pool = c.pool, h.pooled = rt.kv->pooled_layers[L];
            if (c.value_rot) h.n_v = c.n_kv_heads, h.v_width = c.value_dim, h.turn = b->rotary[l.value_rotation], h.turn_half = c.value_dim / 2;
        }
        return launch_head_norms(ctx, st, m->f32, h, p.rows);
    }

    WindowAttn attention_of(const PlainLayer& l) const {
        const tsb_plain_layer& c = l.cfg;
        WindowAttn a;
        a.q = b->q, a.q_stride = b->q_stride, a.out = b->cat, a.out_stride = l.out.cols, a.rows = p.rows_dev;
        a.n_q_heads = c.n_q_heads, a.scale = c.score_scale, a.cap = c.score_cap, a.window = c.window;
        a.slopes = l.slopes, a.chunk = c.chunk, a.keep = c.keep_first, a.pool = c.pool;
        if (c.value_rot) a.turn = b->rotary[l.value_rotation], a.turn_half = c.value_dim / 2;
        if (c.recurrence) a.out_scale = c.attn_scale;
        a.gate = c.head_gate ? b->gate : nullptr;
        if (c.value_gate) a.value_gate = b->value_gate, a.value_gate_stride = b->value_gate_stride;
        if (c.log_bias) a.r1 = l.r1, a.r2 = l.r2;
        if (c.sink) a.sink = l.sink;
        return a;
    }

    cudaError_t attend(int L) const {
        const PlainLayer& l = m->layers[L];
        const int grp = l.cfg.n_q_heads / l.cfg.n_kv_heads;
        WindowAttn a = attention_of(l);
        a.keys = rt.kv->key_layers[L];
        if (a.pool > 0) a.pooled = rt.kv->pooled_layers[L];
        AttnBatch batch;
        if (const AttnBatch* t = plan.find(TILES_ALL, grp, wattn_rows_per_tile(l.head_pad, grp, l.cfg.log_bias != 0))) batch = *t;
        batch.rows = p.rows, batch.rows_per_seq = p.rows_per_seq, batch.max_len = plan.max_len;
        return launch_window_attn(ctx, st, m->f32, a, batch, b->attn_ws);
    }

    // Short portions: queries go to the latents' space, the heads' sums of latents come back from it.
    cudaError_t attend_absorbed(int L, int first, int rows) const {
        const PlainLayer& l = m->layers[L];
        const tsb_plain_layer& c = l.cfg;
        auto product = [&](const PlainMat& w, void* x, int64_t x_stride, void* y, int64_t y_stride, int valid, int step, bool gated) {
            PlainEpi e;
            e.kind = PLAIN_MIXER, e.n_seg = 1;
            PlainSeg& g = e.seg[0];
            g.end = (int)w.rows, g.per = w.group_rows, g.valid = valid, g.step = step, g.p = at(y, first * y_stride), g.stride = y_stride;
            if (gated) g.gate = at(b->value_gate, first * b->value_gate_stride), g.gate_stride = b->value_gate_stride, g.gate_step = l.value_pad;
            return launch_plain_gemm(ctx, st, m->f32, w, at(x, first * x_stride), nullptr, x_stride, b->rows - first, rows, e, b->gemm_ws);
        };
        cudaError_t e = product(l.absorb, b->q, b->q_stride, b->absorbed, b->absorbed_stride, c.kv_rank, l.key_dim, false);
        if (e != cudaSuccess) return e;
        if (m->f32) {
            WindowAttn a = attention_of(l);
            a.keys = rt.kv->key_layers[L], a.q = b->absorbed, a.q_stride = b->absorbed_stride, a.out = b->sums, a.out_stride = b->sums_stride;
            a.value_dim = l.rank_pad, a.value_gate = nullptr;
            AttnBatch batch;
            batch.rows = p.rows, batch.max_len = plan.max_len;
            e = launch_window_attn(ctx, st, true, a, batch, b->attn_ws);
        } else {
            LatentAttn a;
            a.keys = rt.kv->key_layers[L], a.q = b->absorbed, a.q_stride = b->absorbed_stride, a.out = b->sums, a.out_stride = b->sums_stride;
            a.rows = p.rows_dev, a.n_heads = c.n_q_heads, a.value_dim = l.rank_pad, a.scale = c.score_scale, a.sink = c.sink ? l.sink : nullptr;
            const LatentTiling tiling = latent_tiling(ctx, plan, p, l);
            AttnBatch batch;
            if (const AttnBatch* t = plan.find(l.expands ? TILES_LATENT_SHORT : TILES_LATENT, c.n_q_heads, tiling.rows)) batch = *t;
            batch.rows = p.rows, batch.rows_per_seq = p.rows_per_seq, batch.max_len = plan.max_len;
            e = launch_latent_attn(ctx, st, a, batch, tiling, b->attn_ws);
        }
        if (e != cudaSuccess) return e;
        return product(l.lift, b->sums, b->sums_stride, b->cat, l.out.cols, c.value_dim, l.value_pad, c.value_gate != 0);
    }

    // Long portions: keys and values of every visible position, then attention with a key head per query head.
    cudaError_t attend_expanded(int L) const {
        const PlainLayer& l = m->layers[L];
        const tsb_plain_layer& c = l.cfg;
        const int H = c.n_q_heads;
        LatentGather g;
        g.cache = rt.kv->key_layers[L];
        KeyView& w = g.wide;
        w.base = static_cast<uint8_t*>(b->expand.wide), w.page_table = b->expand.table;
        w.kv_heads = H, w.head_dim = l.head_pad, w.elem_bytes = m->elem;
        w.value_off = l.head_pad, w.head_step = l.head_pad + l.value_pad, w.row = H * w.head_step;
        w.page_tokens = EXPAND_PAGE, w.num_pages = b->expand.pages, w.max_seqs = b->expand.max_seqs, w.max_pages_per_seq = b->expand.pages_per_seq;
        for (w.page_shift = 0; 1 << w.page_shift < EXPAND_PAGE;) w.page_shift++;
        g.wide_table = b->expand.table, g.latents = b->expand.latents;
        g.kv_rank = c.kv_rank, g.rot_dim = c.rot_dim, g.key_off = c.head_dim, g.rows = p.rows_dev, g.streams = plan.expanded_dev;
        cudaError_t e = launch_latent_gather(ctx, st, g, (int)plan.expanded.size(), plan.expanded_len);
        if (e != cudaSuccess) return e;
        PlainEpi x;
        x.kind = PLAIN_MIXER, x.n_seg = 2;
        x.seg[0].end = H * c.head_dim, x.seg[0].per = c.head_dim, x.seg[1].end = H * (c.head_dim + c.value_dim), x.seg[1].per = c.value_dim;
        for (PlainSeg& k : x.seg) k.p = w.base, k.stride = w.row, k.step = w.head_step;
        x.seg[1].p = at(w.base, w.value_off);
        e = launch_plain_gemm(ctx, st, false, l.expand, b->expand.latents, nullptr, l.key_dim, b->expand.pages * EXPAND_PAGE, plan.expanded_pages * EXPAND_PAGE, x,
                              b->gemm_ws);
        if (e != cudaSuccess) return e;
        WindowAttn a = attention_of(l);
        a.keys = w, a.value_dim = l.value_pad;
        return launch_window_attn_wide(ctx, st, a, *plan.find(TILES_WIDE, 1, WATTN_WIDE_ROWS), b->attn_ws);
    }

    cudaError_t projection_norms(int L) const {
        const PlainLayer& l = m->layers[L];
        ProjectionNorms n;
        n.raw = b->raw, n.raw_stride = b->raw_stride, n.n_q = l.cfg.n_q_heads, n.n_k = l.cfg.n_kv_heads, n.width = l.cfg.head_dim;
        n.q_weight = l.q_norm, n.k_weight = l.k_norm, n.eps = m->cfg.norm_eps, n.q = b->q, n.q_stride = b->q_stride, n.q_step = l.head_pad;
        n.keys = rt.kv->key_layers[L], n.rows = p.rows_dev;
        if (l.rotation >= 0) n.rot = b->rotary[l.rotation], n.rot_half = l.cfg.rot_dim / 2;
        return launch_projection_norms(ctx, st, m->f32, n, p.rows);
    }

    cudaError_t scan(int L) const {
        const PlainLayer& l = m->layers[L];
        GatedScan g;
        g.gate = b->raw + b->raw_rec, g.gate_stride = b->raw_stride, g.out_gate = b->rec, g.out_gate_stride = b->rec_stride;
        g.out = at(b->cat, l.o_cols), g.out_stride = l.out.cols, g.width = l.cfg.rec_vdim, g.state = b->states.states[L], g.rows = p.rows_dev;
        g.n_rows = p.rows;
        if (cudaError_t e = launch_gated_scan_rows(ctx, st, m->f32, g, plan.by_row); e != cudaSuccess) return e;
        return launch_gated_scan_chunks(ctx, st, m->f32, g, plan.scan_chunks, plan.several_chunks, b->states.scan_sums);
    }

    cudaError_t block_means(int L) const {
        BlockMeans v;
        v.keys = rt.kv->key_layers[L], v.pooled = rt.kv->pooled_layers[L], v.pool = m->layers[L].cfg.pool, v.rows = p.rows_dev;
        return launch_block_means(ctx, st, m->f32, v, p.rows);
    }

    // from the projections to the recurrence's part of b->cat
    cudaError_t recur(int L) const {
        const PlainLayer& l = m->layers[L];
        const tsb_plain_layer& c = l.cfg;
        if (c.recurrence == TSB_REC_MINGRU) return scan(L);
        const int h = c.rec_heads, D = c.rec_dim, E = c.rec_vdim, inner = h * E;
        Recurrence r;
        GatedNorm g;
        r.kind = c.recurrence, r.heads = h, r.dim = D, r.vdim = E, r.gate = b->raw + b->raw_rec, r.gate_stride = b->raw_stride;
        r.q = b->rec, r.q_stride = r.k_stride = r.v_stride = b->rec_stride, r.out = b->rec_out, r.out_stride = b->rec_out_stride;
        r.state = b->states.states[L], r.rows = p.rows_dev, r.n_rows = p.rows;
        g.o = b->rec_out, g.o_stride = b->rec_out_stride, g.width = inner, g.groups = h, g.weight = l.rec_norm, g.weight_n = inner, g.eps = m->cfg.norm_eps;
        g.gate_stride = b->rec_stride, g.out = at(b->cat, l.o_cols), g.out_stride = l.out.cols;
        if (l.mixer != MIX_NONE) g.scale = c.rec_scale;
        if (c.recurrence == TSB_REC_FORGET) {
            r.v = at(b->rec, h * D), r.lower = l.rec_lower;
            g.weight_n = E;
        } else if (c.recurrence == TSB_REC_MLSTM) {
            r.k = at(b->rec, h * D), r.v = at(b->rec, 2 * h * D), r.cap = c.rec_cap, r.q_scale = (float)(1.0 / sqrt((double)D));
            g.post_gate = at(b->rec, 2 * h * D + inner);
        } else {
            ShortConv v;
            v.in = at(b->rec, inner), v.in_stride = b->rec_stride, v.out = b->rec_mixed, v.out_stride = b->rec_mixed_stride, v.channels = (int)rec_conv_channels(c);
            v.taps = c.rec_taps, v.w = l.rec_conv, v.bias = l.rec_conv_bias, v.ring = b->states.rec[L], v.use_before = plan.use_before;
            v.rows = p.rows_dev, v.n_rows = p.rows, v.tiles = plan.runs;
            if (cudaError_t e = launch_short_conv(ctx, st, m->f32, v); e != cudaSuccess) return e;
            r.v = b->rec_mixed, r.k = at(b->rec_mixed, inner), r.q = at(b->rec_mixed, inner + c.rec_groups * D);
            r.q_stride = r.k_stride = r.v_stride = b->rec_mixed_stride, r.heads_per_key = h / c.rec_groups, r.a_log = l.rec_a_log, r.skip = l.rec_skip;
            g.pre_gate = b->rec, g.groups = c.rec_norm_groups;
        }
        const bool chunks = plan.by_chunk.n_portions > 0 && recurrence_chunks_supported(c.recurrence, D, E);
        if (chunks)
            if (cudaError_t e = launch_recurrence_chunks(ctx, st, r, plan.by_chunk); e != cudaSuccess) return e;
        if (cudaError_t e = launch_recurrence_rows(ctx, st, m->f32, r, chunks ? plan.by_row : plan.portions); e != cudaSuccess) return e;
        return launch_gated_norm(ctx, st, m->f32, g, p.rows);
    }

    // The routed feed-forward of b->mix: expert outputs by slot, to be summed by the end of the sublayer.
    cudaError_t route(int L) const {
        const PlainLayer& l = m->layers[L];
        const tsb_plain_layer& c = l.cfg;
        const int slots = p.rows * c.expert_top;
        PlainEpi z;
        z.kind = PLAIN_STORE, z.y = b->router_logits, z.y_stride = c.experts, z.n_valid = c.experts;
        cudaError_t e = matmul(l.router, b->mix, nullptr, b->in_stride, z);
        if (e != cudaSuccess) return e;
        // with many slots per expert the tensor-memory kernel, over gathered rows; with few the weight-streaming one
        const bool tensor = !m->f32 && p.rows > 16 && slots >= 12 * c.experts;
        ExpertRouting r;
        r.logits = b->router_logits, r.logits_stride = c.experts, r.correction = l.correction, r.experts = c.experts, r.top = c.expert_top;
        r.groups = c.expert_groups, r.keep = c.expert_keep, r.rows = p.rows, r.lists = b->lists;
        r.chunk_slots = m->f32 ? EXPERT_CHUNK_F32 : p.rows <= 8 ? 8 : EXPERT_CHUNK_FEW;
        if ((e = launch_route_experts(ctx, st, r)) != cudaSuccess) return e;
        if (tensor && (e = launch_gather_rows(ctx, st, b->mix, b->in_stride * m->elem, b->lists.token_of, slots, b->expert_in, b->in_stride * m->elem)) != cudaSuccess)
            return e;
        PlainExperts x;
        x.n = c.experts, x.slots = slots, x.first = b->lists.first, x.token_of = tensor ? nullptr : b->lists.token_of, x.chunks = b->lists.chunks;
        x.n_chunks = b->lists.n_chunks, x.chunk_slots = r.chunk_slots;
        PlainEpi g;
        g.kind = PLAIN_MIXER, g.pair_row0 = 0, g.n_pairs = l.ffn_pad, g.act = c.act, g.a = b->expert_act, g.a_stride = l.ffn_pad;
        e = launch_plain_gemm_experts(ctx, st, m->f32, tensor, l.ff_in, tensor ? b->expert_in : b->mix, b->in_stride, tensor ? b->expert_rows : b->rows, x, g);
        if (e != cudaSuccess) return e;
        PlainEpi d;
        d.kind = PLAIN_MIXER, d.n_seg = 1, d.seg[0].end = m->cfg.d_model, d.seg[0].p = b->expert_out, d.seg[0].stride = m->cfg.d_model;
        x.token_of = nullptr;
        return launch_plain_gemm_experts(ctx, st, m->f32, tensor, l.ff_out, b->expert_act, l.ffn_pad, b->expert_rows, x, d);
    }

    // The layers of an output-norm model; returns the buffer that holds the stream at the end.
    cudaError_t output_norm_layers(float** stream) const {
        float *x = b->x, *x_next = b->x2;
        SublayerEnd s;
        s.d = m->cfg.d_model, s.groups = std::max(1, m->cfg.norm_groups), s.eps = m->cfg.norm_eps, s.taps = m->cfg.conv_taps, s.use_before = plan.use_before;
        s.out = b->mix, s.out_stride = b->in_stride, s.rows = p.rows_dev, s.n_rows = p.rows, s.tiles = plan.runs;
        // next: the convolution in front of the next sublayer
        auto end = [&](SublayerEnd& v, const float* taps, const RowRing& ring) {
            v.x_in = x, v.x_out = x_next, v.taps_w = taps, v.ring = ring;
            std::swap(x, x_next);
            return launch_sublayer_end(ctx, st, m->f32, v);
        };
        auto first_of = [&](SublayerEnd& v, int L) {  // the end of whatever comes before layer L
            if (L < m->cfg.n_layers) return end(v, m->layers[L].conv1, b->states.conv1.empty() ? RowRing() : b->states.conv1[L]);
            v.taps = 0, v.out = nullptr;
            return end(v, nullptr, RowRing());
        };
        cudaError_t e = plan.use_before ? launch_rings_before(ctx, st, b->states.rings_dev, b->states.n_rings, p.rows_dev, plan.portions) : cudaSuccess;
        if (e != cudaSuccess) return e;
        SublayerEnd t = s;
        t.table = m->embed, t.positions = m->positions, t.n_positions = m->cfg.positions, t.tokens = p.tokens, t.token_stride = p.token_stride, t.vocab = m->cfg.vocab;
        t.embed_scale = m->cfg.embed_scale;
        e = first_of(t, 0);
        for (int L = 0; L < m->cfg.n_layers && e == cudaSuccess; L++) {
            const PlainLayer& l = m->layers[L];
            e = project(L, b->mix, b->mix);
            if (e == cudaSuccess) e = mix(L);
            PlainEpi o;
            o.kind = PLAIN_STORE, o.y = b->y, o.y_stride = m->cfg.d_model, o.n_valid = m->cfg.d_model;
            if (e == cudaSuccess) e = matmul(l.out, b->cat, nullptr, l.out.cols, o);
            SublayerEnd v = s;
            v.y = b->y, v.norm_w = l.gain;
            if (e == cudaSuccess) e = l.cfg.ffn > 0 ? end(v, l.conv2, b->states.conv2.empty() ? RowRing() : b->states.conv2[L]) : first_of(v, L + 1);
            if (e != cudaSuccess || l.cfg.ffn == 0) continue;
            v = s;
            v.norm_w = l.norm2;
            if (l.cfg.experts > 0) {
                e = route(L);
                v.experts = b->expert_out, v.expert_stride = m->cfg.d_model, v.slot_of = b->lists.slot_of, v.weight = b->lists.weight, v.top = l.cfg.expert_top;
            } else {
                PlainEpi g;
                g.kind = PLAIN_MIXER, g.pair_row0 = 0, g.n_pairs = l.ffn_pad, g.act = l.cfg.act, g.a = b->act, g.a_stride = l.ffn_pad;
                e = matmul(l.ff_in, b->mix, b->mix, b->in_stride, g);
                if (e == cudaSuccess) e = matmul(l.ff_out, b->act, nullptr, l.ffn_pad, o);
                v.y = b->y;
            }
            if (e == cudaSuccess) e = first_of(v, L + 1);
        }
        *stream = x;
        return e;
    }

    // from the projections to the heads' outputs, side by side in b->cat
    cudaError_t mix(int L) const {
        const PlainLayer& l = m->layers[L];
        cudaError_t e = cudaSuccess;
        if (l.cfg.recurrence) {
            e = recur(L);
            if (e != cudaSuccess || l.mixer == MIX_NONE) return e;
        }
        if (l.cfg.qk_norm == TSB_NORM_PROJECTION) e = projection_norms(L);
        else if (l.cfg.qk_norm || (l.mixer == MIX_LATENT && l.source == L)) e = head_norms(L);
        // (norms per head see to the blocks before their portions: enough where those are single rows)
        if (e == cudaSuccess && l.cfg.pool > 0 && (plan.longest > 1 || l.cfg.qk_norm != TSB_NORM_HEAD)) e = block_means(L);
        if (e != cudaSuccess) return e;
        if (l.mixer != MIX_LATENT) return attend(L);
        const bool expand = l.expands && !plan.expanded.empty();
        const int first = expand ? plan.short_first : 0, rows = expand ? plan.short_rows : p.rows;
        if (rows > 0) e = attend_absorbed(L, first, rows);  // rows of long portions in between are overwritten below
        return e == cudaSuccess && expand ? attend_expanded(L) : e;
    }

    cudaError_t add_to_stream(const PlainMat& w, const void* x, int64_t stride) const {
        PlainEpi e;
        e.kind = PLAIN_ADD, e.y = b->x, e.y_stride = m->cfg.d_model, e.n_valid = m->cfg.d_model;
        if (m->cfg.post_norm) e.alpha = m->cfg.residual_scale;
        if (m->cfg.pre_norm) e.beta = m->cfg.sublayer_scale;
        return matmul(w, x, nullptr, stride, e);
    }

    // [W_o | W_down] over [heads | feed-forward]: both sublayers read the normed input, and add up in one product
    cudaError_t parallel_layer(int L, bool use_before) const {
        const PlainLayer& l = m->layers[L];
        const tsb_plain_layer& c = l.cfg;
        cudaError_t e = launch_norm_shift(ctx, st, m->f32, b->x, m->cfg.d_model, l.gain, m->cfg.norm_eps, c.token_shift ? l.mu : nullptr, p.rows_dev, p.rows,
                                          b->shift, L, use_before, b->mix, c.ffn > 0 ? b->h : nullptr, b->in_stride);
        if (e == cudaSuccess) e = project(L, b->mix, b->h);
        if (e == cudaSuccess) e = mix(L);
        return e == cudaSuccess ? add_to_stream(l.out, b->cat, l.out.cols) : e;
    }

    // the stream itself is the sublayers' input (b->mix holds it in the compute type), and is normed after each sum
    cudaError_t post_norm_layer(int L) const {
        const PlainLayer& l = m->layers[L];
        cudaError_t e = project(L, b->mix, b->mix);
        if (e == cudaSuccess) e = mix(L);
        if (e == cudaSuccess) e = add_to_stream(l.out, b->cat, l.out.cols);
        auto norm = [&](const float* w) { return launch_post_norm(ctx, st, m->f32, b->x, m->cfg.d_model, w, m->cfg.norm_eps, p.rows, b->mix, b->in_stride); };
        if (e == cudaSuccess) e = norm(l.gain);
        if (e != cudaSuccess || l.cfg.ffn == 0) return e;
        PlainEpi g;
        g.kind = PLAIN_MIXER, g.pair_row0 = 0, g.n_pairs = l.ffn_pad, g.act = l.cfg.act, g.a = b->act, g.a_stride = l.ffn_pad;
        e = matmul(l.ff_in, b->mix, b->mix, b->in_stride, g);
        if (e == cudaSuccess) e = add_to_stream(l.ff_out, b->act, l.ffn_pad);
        return e == cudaSuccess ? norm(l.norm2) : e;
    }

    cudaError_t pre_norm_layer(int L) const {
        const PlainLayer& l = m->layers[L];
        auto norm = [&](const float* w) { return launch_pre_norm(ctx, st, m->f32, b->x, m->cfg.d_model, w, m->cfg.norm_eps, p.rows, b->mix, b->in_stride); };
        cudaError_t e = norm(l.gain);
        if (e == cudaSuccess) e = project(L, b->mix, b->mix);
        if (e == cudaSuccess) e = mix(L);
        if (e == cudaSuccess) e = add_to_stream(l.out, b->cat, l.out.cols);
        if (e != cudaSuccess || l.cfg.ffn == 0) return e;
        e = norm(l.norm2);
        PlainEpi g;
        g.kind = PLAIN_MIXER;
        if (l.cfg.ff_plain) {
            g.n_seg = 1, g.seg[0].end = l.ffn_pad, g.seg[0].act = l.cfg.act, g.seg[0].p = b->act, g.seg[0].stride = l.ffn_pad;
        } else {
            g.pair_row0 = 0, g.n_pairs = l.ffn_pad, g.act = l.cfg.act, g.a = b->act, g.a_stride = l.ffn_pad;
        }
        if (e == cudaSuccess) e = matmul(l.ff_in, b->mix, b->mix, b->in_stride, g);
        return e == cudaSuccess ? add_to_stream(l.ff_out, b->act, l.ffn_pad) : e;
    }
};

cudaError_t plain_forward(tsb_session* s, ModelRt& rt, const Pass& p) {
    tsb_ctx* ctx = s->ctx;
    cudaStream_t st = s->stream;
    const PlainModel* m = rt.model->plain;
    PlainRt* b = rt.plain;
    const int d = m->cfg.d_model;
    const bool post = m->cfg.post_norm != 0;
    PassPlan plan;
    if (plan_pass(s, m, rt, p, plan) != TSB_OK) return cudaErrorMemoryAllocation;
    const Forward f{s, rt, p, ctx, st, m, b, plan};
    cudaError_t e;
#define FW(x)                           \
    do {                                \
        e = (x);                        \
        if (e != cudaSuccess) return e; \
    } while (0)
    const bool use_before = m->any_shift && plan.longest >= b->shift.ring_rows;
    float* x = b->x;
    if (m->cfg.output_norm) {
        FW(f.output_norm_layers(&x));
    } else {
        FW(launch_plain_embed(ctx, st, m->f32, m->embed, m->cfg.vocab, d, p.tokens, p.token_stride, p.rows, m->cfg.embed_scale, x, post ? b->mix : nullptr,
                              b->in_stride));
        if (use_before) FW(launch_shift_before(ctx, st, b->shift, m->cfg.n_layers, p.rows_dev, p.rows));
        for (size_t i = 0; i < m->rotations.size(); i++) {
            const PlainRotation& r = m->rotations[i];
            FW(launch_rotary_table(ctx, st, r.freq, r.dims / 2, r.magnitude, p.rows_dev, p.rows, b->rotary[i]));
        }
        for (int L = 0; L < m->cfg.n_layers; L++) FW(post ? f.post_norm_layer(L) : m->cfg.pre_norm ? f.pre_norm_layer(L) : f.parallel_layer(L, use_before));
    }
    if (p.logits) {
        const bool last = p.last_rows_only && p.rows_per_seq > 1;
        const int n = p.rows_per_seq == 0 ? p.n_want : last ? p.rows / p.rows_per_seq : p.rows;
        if (n > 0) {
            const int32_t* want = p.rows_per_seq == 0 ? p.want_dev : nullptr;
            const int want_first = last ? p.rows_per_seq - 1 : 0, want_step = last ? p.rows_per_seq : 1;
            if (m->cfg.output_norm)
                FW(launch_group_norm_rows(ctx, st, m->f32, x, d, m->final_gain, std::max(1, m->cfg.norm_groups), m->cfg.norm_eps, want, want_first, want_step, n, b->fin,
                                          b->in_stride));
            else
                FW(launch_norm_rows(ctx, st, m->f32, x, d, m->final_gain, m->sequential() ? m->final_gain : nullptr, m->cfg.norm_eps, want, want_first, want_step, n, b->fin, b->in_stride));
            PlainEpi hd;
            hd.kind = PLAIN_STORE, hd.y = static_cast<float*>(p.logits.p), hd.y_stride = p.logits_stride, hd.n_valid = m->cfg.vocab, hd.cap = m->cfg.logit_cap;
            FW(launch_plain_gemm(ctx, st, m->f32, m->head, b->fin, nullptr, b->in_stride, b->fin_rows, n, hd, b->gemm_ws));
        }
    }
#undef FW
    return cudaSuccess;
}

// ------------------------------------------------------------------ rotations
PlainRotation rotation_of(const tsb_plain_layer& c) {
    PlainRotation r;
    r.dims = c.rot_dim, r.base = c.rot_base, r.factor = c.rot_factor, r.original = c.rot_original, r.fast = c.rot_fast, r.slow = c.rot_slow;
    return r;
}
PlainRotation value_rotation_of(const tsb_plain_layer& c) {
    PlainRotation r;
    r.dims = c.value_dim, r.base = c.rot_base;
    return r;
}
int rotation_of(PlainModel* m, const PlainRotation& r) {
    for (size_t i = 0; i < m->rotations.size(); i++) {
        const PlainRotation& o = m->rotations[i];
        if (o.dims == r.dims && o.base == r.base && o.factor == r.factor && o.original == r.original && o.fast == r.fast && o.slow == r.slow) return (int)i;
    }
    m->rotations.push_back(r);
    return (int)m->rotations.size() - 1;
}

int32_t upload_rotation(tsb_ctx* ctx, PlainRotation& r) {
    std::vector<double> freq(r.dims / 2);
    const bool scaled = r.factor > 0 && r.original > 0, linear = r.factor > 0 && !scaled;
    // the pair that turns t times within the original context
    auto pair_with_turns = [&](double t) { return r.dims * log(r.original / (2 * M_PI * t)) / (2 * log(r.base)); };
    const double lo = scaled ? std::max(floor(pair_with_turns(r.fast)), 0.0) : 0;
    const double hi = scaled ? std::min(ceil(pair_with_turns(r.slow)), (double)r.dims - 1) : 0;
    for (int i = 0; i < r.dims / 2; i++) {
        const double f = pow(r.base, -2.0 * i / r.dims);
        const double ramp = scaled ? std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0) : 0;
        freq[i] = linear ? f / r.factor : scaled ? f / r.factor * ramp + f * (1 - ramp) : f;
    }
    r.magnitude = scaled ? (float)(0.1 * log(r.factor) + 1.0) : 1.f;
    if (int32_t rc = tsb_alloc(ctx, freq.size() * sizeof(double), (void**)&r.freq)) return rc;
    TSB_CUDA(ctx, cudaMemcpy(r.freq, freq.data(), freq.size() * sizeof(double), cudaMemcpyHostToDevice));
    return TSB_OK;
}

const ModelFamily PLAIN_FAMILY = {
    "plain-weight", true, false, true, plain_complete, plain_free, plain_weight_bytes, plain_share, plain_runtime_init,
    plain_runtime_free, plain_fill_context, plain_forward,
};

}  // namespace

// what only layers of the output-norm form have
static int32_t check_pre_norm_layer(tsb_ctx* ctx, const tsb_plain_config* cfg, const tsb_plain_layer& l, int i) {
    if (!cfg->pre_norm) {
        TSB_REQUIRE(ctx, !l.keep_first && !l.pool && !l.value_rot && !l.ff_plain && l.act != TSB_ACT_RELU2 && l.recurrence != TSB_REC_MINGRU,
                    "layer %d: prefixes of a window, turning values, feed-forwards without gates and element-wise recurrences go with the pre-norm form", i);
        TSB_REQUIRE(ctx, l.rot_dim == 0 || l.kv_rank > 0, "layer %d: only latent layers and those of the pre-norm form rotate", i);
        return TSB_OK;
    }
    TSB_REQUIRE(ctx, !l.kv_rank && !l.token_shift && !l.head_gate && !l.log_bias && !l.qkv_bias && !l.linear_bias && !l.chunk && !l.experts,
                "layer %d: not a mechanism of the pre-norm form", i);
    TSB_REQUIRE(ctx, l.n_q_heads >= 0 && (l.n_q_heads > 0) != (l.recurrence != 0), "layer %d has one mixer", i);
    if (l.recurrence)
        TSB_REQUIRE(ctx, l.recurrence == TSB_REC_MINGRU && l.rec_heads == 1 && l.rec_dim == 1 && l.rec_vdim > 0, "layer %d: an element-wise recurrence of rec_vdim channels expected", i);
    if (l.n_q_heads == 0) return TSB_OK;
    TSB_REQUIRE(ctx, l.value_dim > 0 && (l.qk_norm == TSB_NORM_HEAD || l.qk_norm == TSB_NORM_PROJECTION), "layer %d: attention has values of its own and normed queries and keys", i);
    TSB_REQUIRE(ctx, l.q_temp_every == 0 || l.qk_norm == TSB_NORM_HEAD, "layer %d: a query temperature goes with norms per head", i);
    TSB_REQUIRE(ctx, l.rot_dim >= 0 && l.rot_dim % 2 == 0 && l.rot_dim <= l.head_dim && ((l.rot_dim == 0 && !l.value_rot) || l.rot_base > 0) && l.rot_factor >= 0,
                "layer %d: an even number of a head's columns is rotated", i);
    TSB_REQUIRE(ctx, !l.value_rot || (l.value_dim % 2 == 0 && l.qk_norm == TSB_NORM_HEAD), "layer %d: values that turn have an even width and go with norms per head", i);
    TSB_REQUIRE(ctx, l.keep_first >= 0 && l.pool >= 0 && !(l.keep_first && l.pool) && ((!l.keep_first && !l.pool) || l.window > 0),
                "layer %d: kept tokens or blocks, before a window", i);
    return TSB_OK;
}

static int32_t check_output_norm_layer(tsb_ctx* ctx, const tsb_plain_config* cfg, const tsb_plain_layer& l, int i) {
    if (!cfg->output_norm) {
        TSB_REQUIRE(ctx, cfg->pre_norm || (!l.recurrence && !l.experts && !l.qkv_bias && !l.linear_bias && !l.chunk && (l.qk_norm == 0 || l.qk_norm == TSB_NORM_HEAD)),
                    "layer %d: recurrences, experts, biases, chunks and projection norms go with the output-norm form", i);
        return TSB_OK;
    }
    TSB_REQUIRE(ctx, !l.kv_rank && !l.token_shift && !l.head_gate && !l.log_bias && l.q_temp_every == 0, "layer %d: not a mechanism of the output-norm form", i);
    TSB_REQUIRE(ctx, l.n_q_heads >= 0 && (l.n_q_heads > 0 || l.recurrence), "layer %d has no mixer", i);
    TSB_REQUIRE(ctx, l.n_q_heads == 0 || l.value_dim > 0, "layer %d: attention has values of its own", i);
    TSB_REQUIRE(ctx, l.chunk >= 0 && !(l.chunk && l.window), "layer %d: a chunk or a window", i);
    TSB_REQUIRE(ctx, l.qk_norm >= 0 && l.qk_norm <= TSB_NORM_PROJECTION && (!l.qkv_bias || l.qk_norm == TSB_NORM_PROJECTION || l.n_q_heads == 0),
                "layer %d: biases go with projection norms", i);
    if (l.recurrence) {
        TSB_REQUIRE(ctx, l.recurrence <= TSB_REC_SSD && l.rec_heads > 0 && l.rec_dim > 0 && l.rec_vdim > 0, "layer %d: bad recurrence", i);
        if (l.rec_dim > REC_MAX_DIM || l.rec_heads > 65535)
            return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "layer %d: recurrent heads of %d rows are outside the kernels", i, l.rec_dim);
        const int64_t inner = (int64_t)l.rec_heads * l.rec_vdim;
        if (inner > 24 * 1024) return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "layer %d: %lld recurrent columns are outside the kernels", i, (long long)inner);
        if (l.recurrence == TSB_REC_SSD) {
            TSB_REQUIRE(ctx, l.rec_groups > 0 && l.rec_heads % l.rec_groups == 0 && l.rec_norm_groups > 0 && inner % l.rec_norm_groups == 0,
                        "layer %d: groups must divide the recurrence's heads and columns", i);
            TSB_REQUIRE(ctx, l.rec_taps > 0 && l.rec_taps <= CONV_MAX_TAPS, "layer %d: a convolution has 1 to %d taps", i, CONV_MAX_TAPS);
        }
        TSB_REQUIRE(ctx, l.recurrence != TSB_REC_MLSTM || l.rec_cap > 0.f, "layer %d: the gates' cap is positive", i);
    }
    TSB_REQUIRE(ctx, l.experts >= 0 && (l.experts == 0 || (l.ffn > 0 && routing_supported(l.experts, l.expert_top, l.expert_groups, l.expert_keep))),
                "layer %d: %d experts in %d groups, %d groups kept and %d experts taken do not fit together", i, l.experts, l.expert_groups, l.expert_keep, l.expert_top);
    return TSB_OK;
}

extern "C" {

int32_t tsb_model_create_plain(tsb_ctx* ctx, const tsb_plain_config* cfg, const tsb_plain_layer* layers, tsb_model** out) {
    if (!ctx || !cfg || !layers || !out) return TSB_ERR_INVALID;
    *out = nullptr;
    TSB_REQUIRE(ctx, cfg->n_layers > 0 && cfg->d_model > 0 && cfg->vocab > 0 && cfg->max_context > 0, "model dimensions must be positive");
    TSB_REQUIRE(ctx, cfg->compute == TSB_BF16 || cfg->compute == TSB_F32, "compute must be TSB_BF16 or TSB_F32");
    TSB_REQUIRE(ctx, cfg->norm_eps >= 0.f, "norm_eps must not be negative");
    const bool f32 = cfg->compute == TSB_F32;
    TSB_REQUIRE(ctx, cfg->norm_groups >= 0 && cfg->conv_taps >= 0 && cfg->positions >= 0, "norm groups, taps and positions must not be negative");
    TSB_REQUIRE(ctx, !cfg->pre_norm || (!cfg->post_norm && !cfg->output_norm), "a model has one form");
    TSB_REQUIRE(ctx, cfg->output_norm ? !cfg->post_norm && cfg->logit_cap <= 0.f : !cfg->norm_groups && !cfg->conv_taps && !cfg->positions,
                "norm groups, convolutions and learned positions go with the output-norm form");
    if (cfg->output_norm && !sublayer_end_supported(cfg->d_model, std::max(1, cfg->norm_groups), cfg->conv_taps))
        return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "width %d in %d norm groups with %d taps is outside the kernels", cfg->d_model, cfg->norm_groups, cfg->conv_taps);
    TSB_REQUIRE(ctx, cfg->positions == 0 || cfg->max_context <= cfg->positions, "a context of %d positions exceeds the learned %d", cfg->max_context, cfg->positions);
    for (int i = 0; i < cfg->n_layers; i++) {
        const tsb_plain_layer& l = layers[i];
        if (int32_t rc = check_output_norm_layer(ctx, cfg, l, i)) return rc;
        if (int32_t rc = check_pre_norm_layer(ctx, cfg, l, i)) return rc;
        TSB_REQUIRE(ctx, l.sink >= 0 && l.sink <= TSB_SINK_ZERO, "layer %d: unknown sink", i);
        if (l.weights_of) {
            TSB_REQUIRE(ctx, l.weights_of > 0 && l.weights_of <= cfg->n_layers && layers[l.weights_of - 1].weights_of == 0, "layer %d: weights_of names a layer with tensors", i);
            tsb_plain_layer same = l;
            same.weights_of = 0;
            TSB_REQUIRE(ctx, memcmp(&same, &layers[l.weights_of - 1], sizeof same) == 0, "layer %d differs from layer %d, whose tensors it uses", i, l.weights_of - 1);
        }
        const bool latent = l.kv_rank > 0;
        if (l.n_q_heads == 0 && l.recurrence) continue;
        TSB_REQUIRE(ctx, l.n_q_heads > 0 && l.head_dim > 0 && (latent || (l.n_kv_heads > 0 && l.n_q_heads % l.n_kv_heads == 0)),
                    "layer %d: query heads must be a positive multiple of the key heads", i);
        TSB_REQUIRE(ctx, l.window >= 0 && l.ffn >= 0 && l.value_dim >= 0 && l.kv_rank >= 0 && l.rot_dim >= 0, "layer %d: sizes must not be negative", i);
        TSB_REQUIRE(ctx, l.act >= TSB_ACT_GELU_TANH && l.act <= TSB_ACT_RELU2, "layer %d: unknown activation", i);
        TSB_REQUIRE(ctx, l.q_temp_every >= 0 && (l.q_temp_every == 0 || l.qk_norm), "layer %d: a query temperature goes with normed queries", i);
        TSB_REQUIRE(ctx, !l.qk_norm || (l.value_dim > 0 && !latent), "layer %d: normed queries and keys go with values of their own", i);
        TSB_REQUIRE(ctx, !cfg->post_norm || !l.token_shift, "layer %d: a token shift goes with the parallel form", i);
        if (latent) {
            TSB_REQUIRE(ctx, cfg->post_norm && l.value_dim > 0 && l.rot_dim % 2 == 0 && (l.rot_dim == 0 || l.rot_base > 0),
                        "layer %d: a latent layer has values, an even rotated part and the post-norm form", i);
            TSB_REQUIRE(ctx, !l.window && l.score_cap <= 0.f && !l.log_bias && !l.head_gate, "layer %d: a latent layer has no window, cap, bias or head gates", i);
            TSB_REQUIRE(ctx, l.kv_source >= 0 && l.kv_source <= i, "layer %d reads the latent of a layer before it", i);
            if (l.kv_source > 0) {
                const tsb_plain_layer& o = layers[l.kv_source - 1];
                TSB_REQUIRE(ctx, o.kv_rank == l.kv_rank && o.rot_dim == l.rot_dim && o.kv_source == 0, "layer %d: layer %d has no latent of this shape", i,
                            l.kv_source - 1);
            }
            int dk = 0, dv = 0;
            if (!latent_attn_dims(l.kv_rank, l.rot_dim, &dk, &dv) || dk > 1024)
                return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "layer %d: latents of %d + %d numbers are outside the attention kernels", i, l.kv_rank, l.rot_dim);
        } else {
            TSB_REQUIRE(ctx, l.kv_source == 0, "layer %d: only latent layers read another layer's rows", i);
            const int head = std::max(l.head_dim, l.value_dim);
            if (!wattn_supported(head, l.n_q_heads / l.n_kv_heads, f32))
                return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "layer %d: head size %d with %d query heads per key head is outside the attention kernels", i, head,
                                l.n_q_heads / l.n_kv_heads);
        }
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
    if (tm->cfg.n_q_heads == 0) tm->cfg.n_q_heads = tm->cfg.n_kv_heads = tm->cfg.head_dim = 1;
    tm->cfg.rms_eps = cfg->norm_eps;
    m->cfg = *cfg, m->f32 = f32, m->elem = f32 ? 4 : 2;
    if (m->cfg.embed_scale == 0.f) m->cfg.embed_scale = 1.f;
    if (m->cfg.sublayer_scale == 0.f) m->cfg.sublayer_scale = 1.f;
    m->d_pad = plain_pad(cfg->d_model, PLAIN_COL_PAD);
    m->head.rows = plain_pad(cfg->vocab, PLAIN_ROW_PAD), m->head.cols = m->d_pad;
    m->layers.resize(cfg->n_layers);
    const int64_t out_rows = plain_pad(cfg->d_model, PLAIN_ROW_PAD);
    for (int i = 0; i < cfg->n_layers; i++) {
        PlainLayer& l = m->layers[i];
        l.cfg = layers[i];
        const tsb_plain_layer& c = l.cfg;
        const int H = c.n_q_heads;
        l.post_norm = m->sequential();
        l.tied = c.weights_of - 1;
        l.mixer = H == 0 ? MIX_NONE : c.kv_rank > 0 ? MIX_LATENT : c.value_dim > 0 ? MIX_KV : MIX_KEYS;
        l.source = c.kv_source > 0 ? c.kv_source - 1 : i;
        m->any_shift |= c.token_shift != 0;
        if (l.mixer == MIX_LATENT) {
            l.head_pad = (int)plain_pad(c.head_dim + c.rot_dim, PLAIN_COL_PAD), l.value_pad = (int)plain_pad(c.value_dim, PLAIN_COL_PAD);
            latent_attn_dims(c.kv_rank, c.rot_dim, &l.key_dim, &l.rank_pad);
            l.expands = !f32 && wattn_wide_supported(l.head_pad, l.value_pad);
            l.rotation = c.rot_dim > 0 ? rotation_of(m, rotation_of(c)) : -1;
            l.absorb.group_rows = (int)plain_pad(c.kv_rank, PLAIN_ROW_PAD), l.absorb.group_cols = l.head_pad;
            l.absorb.rows = (int64_t)H * l.absorb.group_rows, l.absorb.cols = plain_pad(c.head_dim, PLAIN_COL_PAD);
            l.lift.group_rows = (int)plain_pad(c.value_dim, PLAIN_ROW_PAD), l.lift.group_cols = l.rank_pad;
            l.lift.rows = (int64_t)H * l.lift.group_rows, l.lift.cols = plain_pad(c.kv_rank, PLAIN_COL_PAD);
            l.expand.rows = plain_pad((int64_t)H * (c.head_dim + c.value_dim), PLAIN_ROW_PAD), l.expand.cols = l.lift.cols;
        } else if (l.mixer != MIX_NONE) {
            l.head_pad = l.value_pad = wattn_pad_dim(std::max(c.head_dim, c.value_dim), f32);
            if (c.rot_dim > 0) l.rotation = rotation_of(m, rotation_of(c));
            if (c.value_rot) l.value_rotation = rotation_of(m, value_rotation_of(c));
        }
        l.q_rows = H * l.head_pad, l.k_rows = c.n_kv_heads * l.head_pad;
        l.ffn_pad = (int)plain_pad(c.ffn, 64);
        l.in.rows = in_rows(l).rows, l.in.cols = m->d_pad;
        l.o_cols = (int)plain_pad((int64_t)H * l.value_pad, PLAIN_COL_PAD);
        l.rec_cols = (int)plain_pad((int64_t)c.rec_heads * c.rec_vdim * (c.recurrence != 0), PLAIN_COL_PAD);
        l.out.rows = out_rows, l.out.cols = l.o_cols + l.rec_cols + (l.post_norm ? 0 : l.ffn_pad);
        l.ff_in.rows = c.ff_plain ? plain_pad(l.ffn_pad, PLAIN_ROW_PAD) : 2 * (int64_t)l.ffn_pad, l.ff_in.cols = m->d_pad;
        l.ff_out.rows = out_rows, l.ff_out.cols = l.ffn_pad;
        l.router.rows = plain_pad(c.experts, PLAIN_ROW_PAD), l.router.cols = m->d_pad;
    }
    DeviceGuard g(ctx);
    for (PlainLayer& l : m->layers) {
        if (l.tied >= 0) continue;
        if (l.cfg.sink == TSB_SINK_ZERO)
            if (int32_t rc = zeroed(ctx, (size_t)l.cfg.n_q_heads * 4, (void**)&l.sink)) {
                tsb_model_destroy(tm);
                return rc;
            }
        if (!l.cfg.linear_bias) continue;
        std::vector<float> slopes(l.cfg.n_q_heads);
        for (int h = 0; h < l.cfg.n_q_heads; h++) slopes[h] = (float)exp2(-8.0 * (h + 1) / l.cfg.n_q_heads);
        int32_t rc = tsb_alloc(ctx, slopes.size() * 4, (void**)&l.slopes);
        if (rc == TSB_OK && cudaMemcpy(l.slopes, slopes.data(), slopes.size() * 4, cudaMemcpyHostToDevice) != cudaSuccess)
            rc = tsb_fail(ctx, TSB_ERR_CUDA, "uploading slopes failed");
        if (rc) {
            tsb_model_destroy(tm);
            return rc;
        }
    }
    for (PlainRotation& r : m->rotations)
        if (int32_t rc = upload_rotation(ctx, r)) {
            tsb_model_destroy(tm);
            return rc;
        }
    for (int i = 0; i < cfg->n_layers; i++) mirror_layer(m, i);
    *out = tm;
    return TSB_OK;
}

static int32_t set_plain(tsb_model* tm, int32_t layer, int32_t which, int32_t host_type, const void* host, int64_t rows, int64_t cols) {
    if (!tm) return TSB_ERR_INVALID;
    tsb_ctx* ctx = tm->ctx;
    TSB_REQUIRE(ctx, tm->family == &PLAIN_FAMILY, "the model does not hold plain tensors");
    TSB_REQUIRE(ctx, host && (host_type == TSB_BF16 || host_type == TSB_F32), "null data or unknown host type");
    PlainModel* m = tm->plain;
    const int64_t d = m->cfg.d_model, V = m->cfg.vocab;
    PlainLayer* l = nullptr;
    const bool seq = m->sequential();
    if (which >= TSB_P_NORM && which != TSB_P_POSITIONS) {
        TSB_REQUIRE(ctx, layer >= 0 && layer < m->cfg.n_layers, "layer %d outside the model", layer);
        l = &m->layers[layer];
        TSB_REQUIRE(ctx, l->tied < 0, "layer %d uses the tensors of layer %d", layer, l->tied);
    }
    const tsb_plain_layer c = l ? l->cfg : tsb_plain_layer{};
    const bool latent = l && l->mixer == MIX_LATENT, own_latent = latent && c.kv_source == 0;
    const int64_t H = c.n_q_heads, G = c.n_kv_heads, D = c.head_dim, F = c.ffn, E = l && l->mixer != MIX_KEYS ? c.value_dim : D, R = c.kv_rank;
    const int64_t rh = c.recurrence ? c.rec_heads : 0, RD = c.rec_dim, RE = c.rec_vdim, X = std::max(1, c.experts), taps = m->cfg.conv_taps;
    const bool attn = l && l->mixer != MIX_NONE, whole = c.qk_norm == TSB_NORM_PROJECTION;
    const bool forget = c.recurrence == TSB_REC_FORGET, mlstm = c.recurrence == TSB_REC_MLSTM, ssd = c.recurrence == TSB_REC_SSD, gru = c.recurrence == TSB_REC_MINGRU;
    const int64_t channels = rec_conv_channels(c);
    int64_t wr = 1, wc = 1;  // expected shape; -1: no such tensor
    switch (which) {
        case TSB_P_EMBED: case TSB_P_HEAD: wr = V, wc = d; break;
        case TSB_P_FINAL_NORM: case TSB_P_NORM: wc = seq ? d : 1; break;
        case TSB_P_NORM2: wc = seq && F > 0 ? d : -1; break;
        case TSB_P_SHIFT: wc = c.token_shift ? d : -1; break;
        case TSB_P_Q: wr = attn ? H * (D + (latent ? c.rot_dim : 0)) : -1, wc = d; break;
        case TSB_P_K: wr = latent || !attn ? -1 : G * D, wc = d; break;
        case TSB_P_V: wr = l->mixer == MIX_KV ? G * E : -1, wc = d; break;
        case TSB_P_Q_NORM: wc = whole ? H * D : c.qk_norm ? D : -1; break;
        case TSB_P_K_NORM: wc = whole ? G * D : c.qk_norm ? D : -1; break;
        case TSB_P_SINK: wc = c.sink == TSB_SINK_TENSOR ? H : -1; break;
        case TSB_P_HEAD_GATE: wr = c.head_gate ? H : -1, wc = d; break;
        case TSB_P_VALUE_GATE: wr = c.value_gate ? H * E : -1, wc = d; break;
        case TSB_P_R1: case TSB_P_R2: wc = c.log_bias ? H : -1; break;
        case TSB_P_DKV: wr = own_latent ? R + c.rot_dim : -1, wc = d; break;
        case TSB_P_DKV_NORM: wc = own_latent ? R : -1; break;
        case TSB_P_UK: wr = latent ? H * D : -1, wc = R; break;
        case TSB_P_UV: wr = latent ? H * E : -1, wc = R; break;
        case TSB_P_O: wr = d, wc = attn ? H * E : -1; break;
        case TSB_P_FF_GATE: wr = F > 0 && !c.ff_plain ? X * F : -1, wc = d; break;
        case TSB_P_FF_UP: wr = F > 0 ? X * F : -1, wc = d; break;
        case TSB_P_FF_DOWN: wr = X * d, wc = F > 0 ? F : -1; break;
        case TSB_P_POSITIONS: wr = m->cfg.positions > 0 ? m->cfg.positions : -1, wc = d; break;
        case TSB_P_CONV1: wr = d, wc = taps > 0 ? taps : -1; break;
        case TSB_P_CONV2: wr = d, wc = taps > 0 && F > 0 ? taps : -1; break;
        case TSB_P_Q_BIAS: wc = c.qkv_bias ? H * D : -1; break;
        case TSB_P_K_BIAS: wc = c.qkv_bias ? G * D : -1; break;
        case TSB_P_V_BIAS: wc = c.qkv_bias ? G * E : -1; break;
        case TSB_P_ROUTER: wr = c.experts > 0 ? c.experts : -1, wc = d; break;
        case TSB_P_CORRECTION: wc = c.experts > 0 ? c.experts : -1; break;
        case TSB_P_REC_Q: wr = forget || mlstm ? rh * RD : -1, wc = d; break;
        case TSB_P_REC_K: wr = mlstm ? rh * RD : -1, wc = d; break;
        case TSB_P_REC_V: wr = forget || mlstm ? rh * RE : -1, wc = d; break;
        case TSB_P_REC_GATE: wr = mlstm || gru ? rh * RE : -1, wc = d; break;
        case TSB_P_REC_F: wr = forget ? rh * RD : mlstm ? rh : gru ? RE : -1, wc = d; break;
        case TSB_P_REC_F_BIAS: wc = forget ? rh * RD : mlstm ? rh : gru ? RE : -1; break;
        case TSB_P_REC_LOWER: wc = forget ? rh * RD : -1; break;
        case TSB_P_REC_I: wr = mlstm ? rh : gru ? RE : -1, wc = d; break;
        case TSB_P_REC_I_BIAS: wc = mlstm ? rh : gru ? RE : -1; break;
        case TSB_P_REC_NORM: wc = gru ? -1 : forget ? RE : rh > 0 ? rh * RE : -1; break;
        case TSB_P_REC_O: wr = d, wc = rh > 0 ? rh * RE : -1; break;
        case TSB_P_REC_IN: wr = ssd ? rec_typed_rows(c) + rh : -1, wc = d; break;
        case TSB_P_REC_CONV: wr = ssd ? channels : -1, wc = c.rec_taps; break;
        case TSB_P_REC_CONV_BIAS: wc = ssd ? channels : -1; break;
        case TSB_P_REC_DT_BIAS: case TSB_P_REC_A_LOG: case TSB_P_REC_D: wc = ssd ? rh : -1; break;
        default: return tsb_fail(ctx, TSB_ERR_INVALID, "no such tensor (%d)", which);
    }
    TSB_REQUIRE(ctx, wr > 0 && wc > 0, "layer %d has no tensor %d", layer, which);
    TSB_REQUIRE(ctx, rows == wr && cols == wc, "tensor %d of layer %d must be %lld x %lld, got %lld x %lld", which, layer, (long long)wr, (long long)wc,
                (long long)rows, (long long)cols);
    DeviceGuard g(ctx);
    int32_t rc;
    std::vector<uint8_t> v;
    // small f32 vectors
    float** vec = nullptr;
    switch (which) {
        case TSB_P_FINAL_NORM: vec = &m->final_gain; break;
        case TSB_P_NORM: vec = &l->gain; break;
        case TSB_P_NORM2: vec = &l->norm2; break;
        case TSB_P_SHIFT: vec = &l->mu; break;
        case TSB_P_R1: vec = &l->r1; break;
        case TSB_P_R2: vec = &l->r2; break;
        case TSB_P_Q_NORM: vec = &l->q_norm; break;
        case TSB_P_K_NORM: vec = &l->k_norm; break;
        case TSB_P_DKV_NORM: vec = &l->c_norm; break;
        case TSB_P_SINK: vec = &l->sink; break;
        case TSB_P_CORRECTION: vec = &l->correction; break;
        case TSB_P_REC_LOWER: vec = &l->rec_lower; break;
        case TSB_P_REC_NORM: vec = &l->rec_norm; break;
        case TSB_P_REC_CONV_BIAS: vec = &l->rec_conv_bias; break;
        case TSB_P_REC_A_LOG: vec = &l->rec_a_log; break;
        case TSB_P_REC_D: vec = &l->rec_skip; break;
        case TSB_P_CONV1: vec = &l->conv1; break;
        case TSB_P_CONV2: vec = &l->conv2; break;
        case TSB_P_REC_CONV: vec = &l->rec_conv; break;
    }
    uint64_t& set = l ? l->set : m->set;
    const InRows at = l ? in_rows(*l) : InRows();
    // biases: entries of the input matrix's bias, which its epilogue adds
    int64_t bias_at = -1;
    switch (which) {
        case TSB_P_Q_BIAS: bias_at = at.q; break;
        case TSB_P_K_BIAS: bias_at = at.k; break;
        case TSB_P_V_BIAS: bias_at = at.v; break;
        case TSB_P_REC_F_BIAS: bias_at = at.rec_gate + (mlstm ? rh : 0); break;
        case TSB_P_REC_I_BIAS: case TSB_P_REC_DT_BIAS: bias_at = at.rec_gate + (gru ? RE : 0); break;
    }
    if (bias_at >= 0) {
        convert(host, host_type, wc, true, v);
        if (!l->in_bias && (rc = zeroed(ctx, (size_t)l->in.rows * 4, (void**)&l->in_bias))) return rc;
        TSB_CUDA(ctx, cudaMemcpy(l->in_bias + bias_at, v.data(), v.size(), cudaMemcpyHostToDevice));
        set |= 1ull << which;
        return TSB_OK;
    }
    // halves of rotated coordinates -> pairs side by side, in each of `blocks` blocks of `width` items
    auto pair_up = [&](int64_t blocks, int64_t width, int64_t dims, size_t item) {
        std::vector<uint8_t> t(v.size());
        for (int64_t b = 0; b < blocks; b++)
            for (int64_t i = 0; i < width; i++) {
                const int64_t to = i >= dims ? i : i < dims / 2 ? 2 * i : 2 * (i - dims / 2) + 1;
                memcpy(t.data() + (size_t)(b * width + to) * item, v.data() + (size_t)(b * width + i) * item, item);
            }
        v.swap(t);
    };
    const int64_t rotated = l && l->mixer == MIX_KV ? c.rot_dim : 0;
    if (vec) {
        const int64_t n = wr * wc;
        convert(host, host_type, n, true, v);
        if (rotated > 0 && (which == TSB_P_Q_NORM || which == TSB_P_K_NORM)) pair_up(n / D, D, rotated, 4);
        if (wr > 1) {  // taps: [channels, taps] -> [taps][channels]
            std::vector<uint8_t> t(v.size());
            for (int64_t i = 0; i < wr; i++)
                for (int64_t k = 0; k < wc; k++) reinterpret_cast<float*>(t.data())[k * wr + i] = reinterpret_cast<const float*>(v.data())[i * wc + k];
            v.swap(t);
        }
        if (m->shifted_gains() && (which == TSB_P_FINAL_NORM || which == TSB_P_NORM || which == TSB_P_NORM2))  // stored as the distance from one
            for (int64_t i = 0; i < wc; i++) reinterpret_cast<float*>(v.data())[i] += 1.f;
        if (!*vec && (rc = tsb_alloc(ctx, (size_t)n * 4, (void**)vec))) return rc;
        TSB_CUDA(ctx, cudaMemcpy(*vec, v.data(), v.size(), cudaMemcpyHostToDevice));
        set |= 1ull << which;
        return TSB_OK;
    }
    const size_t es = m->elem;
    convert(host, host_type, wr * wc, m->f32, v);
    if (rotated > 0 && (which == TSB_P_Q || which == TSB_P_K)) pair_up(wr / D, D, rotated, (size_t)d * es);
    if (c.value_rot && which == TSB_P_V) pair_up(G, E, E, (size_t)d * es);
    if (c.value_rot && which == TSB_P_O) pair_up(d * H, E, E, es);
    if (which == TSB_P_EMBED || which == TSB_P_POSITIONS) {
        void*& table = which == TSB_P_EMBED ? m->embed : m->positions;
        if (!table && (rc = tsb_alloc(ctx, v.size(), &table))) return rc;
        TSB_CUDA(ctx, cudaMemcpy(table, v.data(), v.size(), cudaMemcpyHostToDevice));
        set |= 1ull << which;
        return TSB_OK;
    }
    // block of n_rows x n_cols of the host tensor (hw columns wide) at (hr, hc) -> the packed matrix at (dr, dc)
    auto put_from = [&](PlainMat& mat, const uint8_t* data, int64_t hw, int64_t dr, int64_t dc, int64_t hr, int64_t hc, int64_t n_rows, int64_t n_cols) -> int32_t {
        if (!mat.data)
            if (int32_t r = zeroed(ctx, (size_t)mat.rows * (l && (&mat == &l->ff_in || &mat == &l->ff_out) ? X : 1) * mat.cols * es, &mat.data)) return r;
        const size_t pitch = (size_t)mat.cols * es;
        TSB_CUDA(ctx, cudaMemcpy2D(static_cast<uint8_t*>(mat.data) + (size_t)dr * pitch + (size_t)dc * es, pitch, data + ((size_t)hr * hw + hc) * es, (size_t)hw * es,
                                   (size_t)n_cols * es, (size_t)n_rows, cudaMemcpyHostToDevice));
        return TSB_OK;
    };
    auto put = [&](PlainMat& mat, int64_t dr, int64_t dc, int64_t hr, int64_t hc, int64_t n_rows, int64_t n_cols) {
        return put_from(mat, v.data(), wc, dr, dc, hr, hc, n_rows, n_cols);
    };
#define PUT(...)                                  \
    do {                                          \
        if ((rc = put(__VA_ARGS__))) return rc;   \
    } while (0)
    // rows hr + i and hr + half + i of the host tensor are the coordinates of pair `first` + i
    auto put_pairs = [&](int64_t first, int64_t hr, int64_t half) -> int32_t {
        for (int64_t i = 0; i < half;) {
            const int64_t p = first + i, n = std::min<int64_t>(8 - p % 8, half - i), dr = at.pairs + p / 8 * 16 + p % 8;
            int32_t r = put(l->in, dr, 0, hr + i, 0, n, d);
            if (r == TSB_OK) r = put(l->in, dr + 8, 0, hr + half + i, 0, n, d);
            if (r) return r;
            i += n;
        }
        return TSB_OK;
    };
    switch (which) {
        case TSB_P_HEAD: PUT(m->head, 0, 0, 0, 0, wr, wc); break;
        case TSB_P_Q:
            if (l->mixer == MIX_KV) {
                PUT(l->in, at.q, 0, 0, 0, wr, d);
            } else {
                const int64_t step = latent ? D : l->head_pad, from = D + c.rot_dim;
                for (int64_t h = 0; h < H; h++) {
                    PUT(l->in, at.q + h * step, 0, h * from, 0, D, d);
                    if ((rc = put_pairs(h * (c.rot_dim / 2), h * from + D, c.rot_dim / 2))) return rc;
                }
            }
            break;
        case TSB_P_K:
            if (l->mixer == MIX_KV) PUT(l->in, at.k, 0, 0, 0, wr, d);
            else for (int64_t h = 0; h < G; h++) PUT(l->in, at.k + h * l->head_pad, 0, h * D, 0, D, d);
            break;
        case TSB_P_V: PUT(l->in, at.v, 0, 0, 0, wr, d); break;
        case TSB_P_DKV:
            PUT(l->in, at.k, 0, 0, 0, R, d);
            if ((rc = put_pairs(H * (c.rot_dim / 2), R, c.rot_dim / 2))) return rc;
            break;
        case TSB_P_HEAD_GATE: PUT(l->in, at.head_gate, 0, 0, 0, H, d); break;
        case TSB_P_VALUE_GATE: PUT(l->in, at.value_gate, 0, 0, 0, wr, d); break;
        case TSB_P_UK: {
            std::vector<uint8_t> t(v.size());  // head by head transposed: [H][R][D]
            auto transpose = [&](const auto* from, auto* to) {
                for (int64_t h = 0; h < H; h++)
                    for (int64_t i = 0; i < D; i++)
                        for (int64_t k = 0; k < R; k++) to[(h * R + k) * D + i] = from[(h * D + i) * R + k];
            };
            if (m->f32) transpose((const uint32_t*)v.data(), (uint32_t*)t.data());
            else transpose((const uint16_t*)v.data(), (uint16_t*)t.data());
            for (int64_t h = 0; h < H; h++)
                if ((rc = put_from(l->absorb, t.data(), D, h * l->absorb.group_rows, 0, h * R, 0, R, D))) return rc;
            if (l->expands) PUT(l->expand, 0, 0, 0, 0, H * D, R);
            break;
        }
        case TSB_P_UV:
            for (int64_t h = 0; h < H; h++) PUT(l->lift, h * l->lift.group_rows, 0, h * E, 0, E, R);
            if (l->expands) PUT(l->expand, H * D, 0, 0, 0, H * E, R);
            break;
        case TSB_P_O:
            for (int64_t h = 0; h < H; h++) PUT(l->out, 0, h * l->value_pad, 0, h * E, d, E);
            break;
        case TSB_P_FF_GATE: case TSB_P_FF_UP: {
            if (c.ff_plain) {
                PUT(l->ff_in, 0, 0, 0, 0, F, d);
                break;
            }
            const int64_t row0 = (seq ? 0 : at.pairs) + (which == TSB_P_FF_UP ? 8 : 0);
            for (int64_t x = 0; x < X; x++) {
                PlainMat& mat = seq ? l->ff_in : l->in;
                int64_t i = 0;
                if (mat.data && mat.cols == d && F >= 16) {  // whole groups of eight rows at once
                    i = F / 8 * 8;
                    TSB_CUDA(ctx, cudaMemcpy2D(static_cast<uint8_t*>(mat.data) + (size_t)(x * mat.rows * seq + row0) * d * es, (size_t)16 * d * es,
                                               v.data() + (size_t)x * F * d * es, (size_t)8 * d * es, (size_t)8 * d * es, (size_t)F / 8, cudaMemcpyHostToDevice));
                }
                for (; i < F; i += 8) PUT(mat, x * mat.rows * seq + row0 + 2 * i, 0, x * F + i, 0, std::min<int64_t>(8, F - i), d);
            }
            break;
        }
        case TSB_P_FF_DOWN:
            for (int64_t x = 0; x < X; x++) PUT(seq ? l->ff_out : l->out, x * l->ff_out.rows, seq ? 0 : l->o_cols, x * d, 0, d, F);
            break;
        case TSB_P_ROUTER: PUT(l->router, 0, 0, 0, 0, wr, d); break;
        // the recurrence's vectors: queries, keys and values (MLSTM), values, output gates; SSD: z | x | B | C, its steps with the gates
        case TSB_P_REC_Q: PUT(l->in, at.rec, 0, 0, 0, wr, d); break;
        case TSB_P_REC_K: PUT(l->in, at.rec + rh * RD, 0, 0, 0, wr, d); break;
        case TSB_P_REC_V: PUT(l->in, at.rec + (mlstm ? 2 : 1) * rh * RD, 0, 0, 0, wr, d); break;
        case TSB_P_REC_GATE: PUT(l->in, at.rec + (gru ? 0 : 2 * rh * RD + rh * RE), 0, 0, 0, wr, d); break;
        case TSB_P_REC_I: PUT(l->in, at.rec_gate + (gru ? RE : 0), 0, 0, 0, wr, d); break;  // MINGRU: z, then the candidate
        case TSB_P_REC_F: PUT(l->in, at.rec_gate + (mlstm ? rh : 0), 0, 0, 0, wr, d); break;
        case TSB_P_REC_IN: PUT(l->in, at.rec, 0, 0, 0, wr, d); break;
        case TSB_P_REC_O: PUT(l->out, 0, l->o_cols, 0, 0, d, rh * RE); break;
    }
#undef PUT
    set |= 1ull << which;
    return TSB_OK;
}

int32_t tsb_model_set_plain(tsb_model* tm, int32_t layer, int32_t which, int32_t host_type, const void* host, int64_t rows, int64_t cols) {
    const int32_t rc = set_plain(tm, layer, which, host_type, host, rows, cols);
    if (rc == TSB_OK && which >= TSB_P_NORM && which != TSB_P_POSITIONS) mirror_layer(tm->plain, layer);
    return rc;
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
        if (rc || rows * cols == 0) return;
        if (!*p && (rc = tsb_alloc(ctx, (size_t)rows * cols * (f32 ? 4 : 2), p))) return;
        if (f32) fill_plain_kernel<float><<<1024, 256>>>((float*)*p, rows, cols, valid, mid, amp, sd);
        else fill_plain_kernel<__nv_bfloat16><<<1024, 256>>>((__nv_bfloat16*)*p, rows, cols, valid, mid, amp, sd);
        sd = sd * 1664525u + 1013904223u;
    };
    auto matrix = [&](PlainMat& w, int64_t valid, float gain) { fill(&w.data, m->f32, w.rows, w.cols, valid, 0.f, gain * sqrtf(3.f / (float)valid)); };
    auto vector = [&](float*& p, int64_t n, float mid, float amp) { fill((void**)&p, true, 1, n, n, mid, amp); };
    const int64_t d = m->cfg.d_model, gains = m->sequential() ? d : 1;
    fill(&m->embed, m->f32, m->cfg.vocab, d, d, 0.f, 1.7f);
    matrix(m->head, d, 1.f);
    vector(m->final_gain, gains, 1.f, 0.f);
    if (m->cfg.positions > 0) fill(&m->positions, m->f32, m->cfg.positions, d, d, 0.f, 0.3f);
    m->set = ~0ull;
    for (PlainLayer& l : m->layers) {
        const tsb_plain_layer& c = l.cfg;
        if (l.tied >= 0) continue;
        matrix(l.in, d, 1.f);
        matrix(l.out, l.out.cols, 0.5f);
        vector(l.gain, gains, 1.f, 0.f);
        if (c.token_shift) vector(l.mu, d, 0.5f, 0.4f);
        if (c.log_bias) vector(l.r1, c.n_q_heads, 1.f, 0.5f), vector(l.r2, c.n_q_heads, 0.3f, 0.2f);
        if (c.sink == TSB_SINK_TENSOR) vector(l.sink, c.n_q_heads, 0.f, 1.f);
        const int64_t whole = c.qk_norm == TSB_NORM_PROJECTION ? 1 : 0;
        if (c.qk_norm) vector(l.q_norm, c.head_dim * (whole ? c.n_q_heads : 1), 1.f, 0.2f), vector(l.k_norm, c.head_dim * (whole ? c.n_kv_heads : 1), 1.f, 0.2f);
        auto experts = [&](PlainMat& w, int64_t valid, float gain) {
            fill(&w.data, m->f32, w.rows * std::max(1, c.experts), w.cols, valid, 0.f, gain * sqrtf(3.f / (float)valid));
        };
        if (l.post_norm && c.ffn > 0) experts(l.ff_in, d, 1.f), experts(l.ff_out, c.ffn, 0.5f), vector(l.norm2, d, 1.f, 0.f);
        if (c.experts > 0) matrix(l.router, d, 1.f), vector(l.correction, c.experts, 0.f, 0.1f);
        if (m->cfg.conv_taps > 0) vector(l.conv1, d * m->cfg.conv_taps, 0.f, 0.3f);
        if (m->cfg.conv_taps > 0 && c.ffn > 0) vector(l.conv2, d * m->cfg.conv_taps, 0.f, 0.3f);
        if (c.qkv_bias || c.recurrence) vector(l.in_bias, l.in.rows, 0.f, 0.2f);
        if (c.recurrence && c.recurrence != TSB_REC_MINGRU) {
            const int64_t inner = (int64_t)c.rec_heads * c.rec_vdim;
            vector(l.rec_norm, c.recurrence == TSB_REC_FORGET ? c.rec_vdim : inner, 1.f, 0.2f);
            if (c.recurrence == TSB_REC_FORGET) vector(l.rec_lower, (int64_t)c.rec_heads * c.rec_dim, 0.5f, 0.4f);
            if (c.recurrence == TSB_REC_SSD)
                vector(l.rec_conv, rec_conv_channels(c) * c.rec_taps, 0.f, 0.5f), vector(l.rec_conv_bias, rec_conv_channels(c), 0.f, 0.2f),
                    vector(l.rec_a_log, c.rec_heads, 0.f, 1.f), vector(l.rec_skip, c.rec_heads, 1.f, 0.2f);
        }
        if (l.mixer == MIX_LATENT) {
            vector(l.c_norm, c.kv_rank, 1.f, 0.f);
            matrix(l.absorb, c.head_dim, 1.f), matrix(l.lift, c.kv_rank, 1.f);
            if (l.expands) matrix(l.expand, c.kv_rank, 1.f);
        }
        l.set = ~0ull;
    }
    for (int i = 0; i < m->cfg.n_layers; i++) mirror_layer(m, i);
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
    TSB_REQUIRE(ctx, act >= TSB_ACT_GELU_TANH && act <= TSB_ACT_RELU2, "unknown activation");
    DeviceGuard g(ctx);
    PlainEpi e;
    e.kind = PLAIN_MIXER, e.pair_row0 = 0, e.n_pairs = n_pairs, e.act = act, e.a = a, e.a_stride = a_stride;
    TSB_CUDA(ctx, launch_plain_gemm(ctx, (cudaStream_t)s, type == TSB_F32, PlainMat{const_cast<void*>(w), rows, cols}, x, x, cols, x_rows, tokens, e,
                                    workspace));
    return TSB_OK;
}

int32_t tsb_plain_gemm_act(tsb_ctx* ctx, tsb_stream s, int32_t type, const void* w, int64_t rows, int64_t cols, const void* x, int32_t x_rows, int32_t tokens,
                           void* y, int64_t y_stride, int32_t n_valid, int32_t act, void* workspace) {
    if (!ctx) return TSB_ERR_INVALID;
    int32_t rc = check_gemm(ctx, type, w, rows, cols, x, x_rows, tokens, workspace);
    if (rc) return rc;
    TSB_REQUIRE(ctx, y && n_valid > 0 && n_valid <= rows && y_stride >= n_valid, "bad output");
    TSB_REQUIRE(ctx, act >= TSB_ACT_GELU_TANH && act <= TSB_ACT_RELU2, "unknown activation");
    DeviceGuard g(ctx);
    PlainEpi e;
    e.kind = PLAIN_MIXER, e.n_seg = 1, e.seg[0].end = n_valid, e.seg[0].act = act, e.seg[0].p = y, e.seg[0].stride = y_stride;
    TSB_CUDA(ctx, launch_plain_gemm(ctx, (cudaStream_t)s, type == TSB_F32, PlainMat{const_cast<void*>(w), rows, cols}, x, nullptr, cols, x_rows, tokens, e, workspace));
    return TSB_OK;
}

int32_t tsb_plain_gemm_add(tsb_ctx* ctx, tsb_stream s, int32_t type, const void* w, int64_t rows, int64_t cols, const void* x, int32_t x_rows, int32_t tokens,
                           float* y, int64_t y_stride, int32_t n_valid, float alpha, float beta, void* workspace) {
    if (!ctx) return TSB_ERR_INVALID;
    int32_t rc = check_gemm(ctx, type, w, rows, cols, x, x_rows, tokens, workspace);
    if (rc) return rc;
    TSB_REQUIRE(ctx, y && n_valid > 0 && n_valid <= rows && y_stride >= n_valid, "bad output");
    DeviceGuard g(ctx);
    PlainEpi e;
    e.kind = PLAIN_ADD, e.y = y, e.y_stride = y_stride, e.n_valid = n_valid, e.alpha = alpha, e.beta = beta;
    TSB_CUDA(ctx, launch_plain_gemm(ctx, (cudaStream_t)s, type == TSB_F32, PlainMat{const_cast<void*>(w), rows, cols}, x, nullptr, cols, x_rows, tokens, e, workspace));
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
    TSB_REQUIRE(ctx, wattn_pad_dim(head_dim, type == TSB_F32) == head_dim, "head size %d is not one the attention kernels work on", head_dim);
    return tsb_kv_create_plain(ctx, type, layers, kv_heads, head_dim, 0, page_tokens, num_pages, max_seqs, max_pages_per_seq, out);
}

int32_t tsb_kv_create_plain(tsb_ctx* ctx, int32_t type, int32_t layers, int32_t kv_heads, int32_t key_dim, int32_t value_dim, int32_t page_tokens,
                            int32_t num_pages, int32_t max_seqs, int32_t max_pages_per_seq, tsb_kv** out) {
    return tsb_kv_create_blocks(ctx, type, layers, kv_heads, key_dim, value_dim, 0, page_tokens, num_pages, max_seqs, max_pages_per_seq, out);
}

int32_t tsb_kv_create_blocks(tsb_ctx* ctx, int32_t type, int32_t layers, int32_t kv_heads, int32_t key_dim, int32_t value_dim, int32_t pool, int32_t page_tokens,
                             int32_t num_pages, int32_t max_seqs, int32_t max_pages_per_seq, tsb_kv** out) {
    if (!ctx || !out) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, (type == TSB_BF16 || type == TSB_F32) && layers > 0 && kv_heads > 0 && pool >= 0, "unknown type or bad sizes");
    std::vector<KeyLayerShape> shapes;
    for (int l = 0; l < layers; l++) shapes.push_back({kv_heads, key_dim, value_dim, l, pool});
    return kv_create_keys(ctx, layers, shapes.data(), type == TSB_F32 ? 4 : 2, page_tokens, num_pages, max_seqs, max_pages_per_seq, out);
}

// The tiles of a batch of unequal portions, uploaded behind the launches before it: launch(batch) with them, then freed.
static int32_t with_tiles(tsb_ctx* ctx, cudaStream_t st, const std::vector<AttnTile>& small, const std::vector<AttnTile>& large, AttnBatch b,
                          const std::function<cudaError_t(const AttnBatch&)>& launch) {
    // a captured copy would read the list again at every replay, when it is gone
    cudaStreamCaptureStatus capture = cudaStreamCaptureStatusNone;
    TSB_CUDA(ctx, cudaStreamIsCapturing(st, &capture));
    if (capture != cudaStreamCaptureStatusNone) return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "portions of unequal length cannot be captured in a graph");
    std::vector<AttnTile> all = small;
    all.insert(all.end(), large.begin(), large.end());
    AttnTile* dev = nullptr;
    TSB_CUDA(ctx, cudaMallocAsync((void**)&dev, all.size() * sizeof(AttnTile), st));
    cudaError_t e = cudaMemcpyAsync(dev, all.data(), all.size() * sizeof(AttnTile), cudaMemcpyHostToDevice, st);
    b.n_small = (int)small.size(), b.n_large = (int)large.size(), b.small = dev, b.large = dev + b.n_small;
    if (e == cudaSuccess) e = launch(b);
    cudaError_t e2 = cudaFreeAsync(dev, st);
    TSB_CUDA(ctx, e);
    TSB_CUDA(ctx, e2);
    return TSB_OK;
}

int32_t tsb_window_attention(tsb_ctx* ctx, tsb_stream s, tsb_kv* keys, int32_t layer, const void* q, int64_t q_stride, void* out, int64_t out_stride,
                             const tsb_row_desc* rows_dev, const int32_t* group_rows, int32_t n_groups, int32_t n_q_heads, float scale, float cap,
                             const float* r1, const float* r2, const float* gate, int32_t window, int32_t max_len, void* scratch) {
    tsb_attention_extras x{};
    x.cap = cap, x.r1 = r1, x.r2 = r2, x.head_gate = gate, x.window = window;
    return tsb_plain_attention(ctx, s, keys, layer, q, q_stride, out, out_stride, rows_dev, group_rows, n_groups, n_q_heads, scale, &x, max_len, scratch);
}

int32_t tsb_plain_attention(tsb_ctx* ctx, tsb_stream s, tsb_kv* keys, int32_t layer, const void* q, int64_t q_stride, void* out, int64_t out_stride,
                            const tsb_row_desc* rows_dev, const int32_t* group_rows, int32_t n_groups, int32_t n_q_heads, float scale,
                            const tsb_attention_extras* extras, int32_t max_len, void* scratch) {
    if (!ctx || !keys) return TSB_ERR_INVALID;
    const tsb_attention_extras x = extras ? *extras : tsb_attention_extras{};
    TSB_REQUIRE(ctx, !keys->key_layers.empty() && layer >= 0 && layer < (int)keys->key_layers.size(), "a plain cache and one of its layers expected");
    TSB_REQUIRE(ctx, q && out && rows_dev && group_rows && n_groups > 0 && scratch && (x.r1 == nullptr) == (x.r2 == nullptr) && x.window >= 0 &&
                         x.chunk >= 0 && !(x.window && x.chunk) && !(x.r1 && x.slopes), "bad arguments");
    const KeyView& kv = keys->key_layers[layer];
    TSB_REQUIRE(ctx, x.keep >= 0 && ((x.keep == 0 && !x.blocks) || (x.window > 0 && kv.value_off > 0 && !x.r1 && !x.slopes && !(x.keep && x.blocks))) &&
                         (!x.blocks || keys->pool_sizes[layer] > 0), "a prefix goes with a window over values of their own and no distance bias");
    const bool f32 = kv.elem_bytes == 4;
    const int vd = kv.value_off ? kv.head_step - kv.value_off : kv.head_dim;
    const bool wide = vd != kv.head_dim;  // keys and values of different widths: the many-query kernel alone takes them
    const int grp = n_q_heads / kv.kv_heads;
    TSB_REQUIRE(ctx, n_q_heads > 0 && n_q_heads % kv.kv_heads == 0 && (f32 ? kv.head_dim <= 1024 && vd <= 512 : wide ? grp == 1 && wattn_wide_supported(kv.head_dim, vd) && !x.r1
                     : wattn_supported(kv.head_dim, grp, false) && wattn_pad_dim(kv.head_dim, false) == kv.head_dim),
                "query heads must be a multiple of the key heads, at most %d per key head, and the head size one the kernels take", WATTN_LARGE_Q);
    TSB_REQUIRE(ctx, (uintptr_t)q % 32 == 0 && (uintptr_t)out % 32 == 0 && q_stride % 16 == 0 && out_stride % 16 == 0 &&
                         q_stride >= (int64_t)n_q_heads * kv.head_dim && out_stride >= (int64_t)n_q_heads * vd,
                "q and out rows hold every head and start on 32-byte boundaries (strides a multiple of 16)");
    TSB_REQUIRE(ctx, !x.turn || (x.turn_half > 0 && 2 * x.turn_half <= vd && (uintptr_t)x.turn % 8 == 0 && !wide), "turned columns are a head's first ones");
    TSB_REQUIRE(ctx, !x.value_gate || ((uintptr_t)x.value_gate % 32 == 0 && x.value_gate_stride % 16 == 0 && x.value_gate_stride >= (int64_t)n_q_heads * vd),
                "rows of value gates hold every head and start on 32-byte boundaries");
    cudaStream_t st = (cudaStream_t)s;
    DeviceGuard g(ctx);
    WindowAttn a;
    a.keys = kv, a.q = q, a.q_stride = q_stride, a.out = out, a.out_stride = out_stride, a.gate = x.head_gate, a.rows = rows_dev;
    a.n_q_heads = n_q_heads, a.scale = scale, a.cap = x.cap, a.r1 = x.r1, a.r2 = x.r2, a.window = x.window;
    a.sink = x.sink, a.value_gate = x.value_gate, a.value_gate_stride = x.value_gate_stride, a.value_dim = vd;
    a.slopes = x.slopes, a.chunk = x.chunk, a.out_scale = x.out_scale == 0.f ? 1.f : x.out_scale;
    a.keep = x.keep, a.turn = reinterpret_cast<const float2*>(x.turn), a.turn_half = x.turn ? x.turn_half : 0;
    if (x.blocks) a.pool = keys->pool_sizes[layer], a.pooled = keys->pooled_layers[layer];
    AttnBatch b;
    b.max_len = max_len;
    bool uniform = true;
    for (int i = 0; i < n_groups; i++) {
        TSB_REQUIRE(ctx, group_rows[i] > 0, "every stream of the batch has rows");
        b.rows += group_rows[i];
        uniform &= group_rows[i] == group_rows[0];
    }
    if (f32 || uniform) {
        if (uniform) b.rows_per_seq = group_rows[0];
        TSB_CUDA(ctx, wide && !f32 ? launch_window_attn_wide(ctx, st, a, b, scratch) : launch_window_attn(ctx, st, f32, a, b, scratch));
        return TSB_OK;
    }
    const int rpt = wide ? WATTN_WIDE_ROWS : wattn_rows_per_tile(kv.head_dim, grp, x.r1 != nullptr);
    std::vector<AttnTile> small, large;
    for (int i = 0, r = 0; i < n_groups; r += group_rows[i], i++) {
        if (!wide && group_rows[i] * grp <= WATTN_SMALL_Q) {
            small.push_back({r, group_rows[i]});
            b.small_queries = std::max(b.small_queries, group_rows[i] * grp);
        } else {
            for (int k = 0; k < group_rows[i]; k += rpt) large.push_back({r + k, std::min(rpt, group_rows[i] - k)});
        }
    }
    return with_tiles(ctx, st, small, large, b, [&](const AttnBatch& t) {
        return wide ? launch_window_attn_wide(ctx, st, a, t, scratch) : launch_window_attn(ctx, st, false, a, t, scratch);
    });
}

int32_t tsb_latent_attention(tsb_ctx* ctx, tsb_stream s, tsb_kv* cache, int32_t layer, const void* q, int64_t q_stride, void* out, int64_t out_stride,
                             const tsb_row_desc* rows_dev, const int32_t* group_rows, int32_t n_groups, int32_t n_heads, int32_t value_dim, float scale,
                             const float* sink, int32_t max_len, void* scratch) {
    if (!ctx || !cache) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, !cache->key_layers.empty() && layer >= 0 && layer < (int)cache->key_layers.size(), "a plain cache and one of its layers expected");
    const KeyView& kv = cache->key_layers[layer];
    int key_pad = 0, value_pad = 0;
    TSB_REQUIRE(ctx, q && out && rows_dev && group_rows && n_groups > 0 && scratch && n_heads > 0 && kv.kv_heads == 1 && kv.value_off == 0, "bad arguments");
    TSB_REQUIRE(ctx, latent_attn_dims(value_dim, kv.head_dim - value_dim, &key_pad, &value_pad) && value_pad == value_dim && key_pad == kv.head_dim,
                "a row of %d numbers, the first %d of them the value, is not one the kernels work on", kv.head_dim, value_dim);
    TSB_REQUIRE(ctx, (uintptr_t)q % 32 == 0 && (uintptr_t)out % 32 == 0 && q_stride % 16 == 0 && out_stride % 16 == 0 &&
                         q_stride >= (int64_t)n_heads * kv.head_dim && out_stride >= (int64_t)n_heads * value_dim,
                "q and out rows hold every head and start on 32-byte boundaries (strides a multiple of 16)");
    cudaStream_t st = (cudaStream_t)s;
    DeviceGuard g(ctx);
    AttnBatch b;
    b.max_len = max_len;
    int most = 0;
    bool uniform = true;
    for (int i = 0; i < n_groups; i++) {
        TSB_REQUIRE(ctx, group_rows[i] > 0, "every stream of the batch has rows");
        b.rows += group_rows[i], most = std::max(most, group_rows[i]);
        uniform &= group_rows[i] == group_rows[0];
    }
    if (kv.elem_bytes == 4) {
        WindowAttn a;
        a.keys = kv, a.q = q, a.q_stride = q_stride, a.out = out, a.out_stride = out_stride, a.rows = rows_dev, a.n_q_heads = n_heads, a.scale = scale;
        a.sink = sink, a.value_dim = value_dim;
        TSB_CUDA(ctx, launch_window_attn(ctx, st, true, a, b, scratch));
        return TSB_OK;
    }
    LatentAttn a;
    a.keys = kv, a.q = q, a.q_stride = q_stride, a.out = out, a.out_stride = out_stride, a.rows = rows_dev, a.n_heads = n_heads, a.value_dim = value_dim;
    a.scale = scale, a.sink = sink;
    const LatentTiling tiling = latent_attn_tiling(ctx, n_heads, most, b.rows, max_len);
    if (uniform) {
        b.rows_per_seq = most;
        TSB_CUDA(ctx, launch_latent_attn(ctx, st, a, b, tiling, scratch));
        return TSB_OK;
    }
    const int rpt = tiling.rows;
    std::vector<AttnTile> tiles;
    for (int i = 0, r = 0; i < n_groups; r += group_rows[i], i++)
        for (int k = 0; k < group_rows[i]; k += rpt) tiles.push_back({r + k, std::min(rpt, group_rows[i] - k)});
    return with_tiles(ctx, st, tiles, {}, b, [&](const AttnBatch& t) { return launch_latent_attn(ctx, st, a, t, tiling, scratch); });
}

int32_t tsb_plain_gemm_heads(tsb_ctx* ctx, tsb_stream s, int32_t type, const void* w, int32_t heads, int32_t head_rows, int64_t cols, const void* x,
                             int64_t x_stride, int32_t x_step, int32_t x_rows, int32_t tokens, void* y, int64_t y_stride, int32_t y_step, int32_t n_valid,
                             const void* gate, int64_t gate_stride, int32_t gate_step, void* workspace) {
    if (!ctx) return TSB_ERR_INVALID;
    int32_t rc = check_gemm(ctx, type, w, (int64_t)heads * head_rows, cols, x, x_rows, tokens, workspace);
    if (rc) return rc;
    TSB_REQUIRE(ctx, heads > 0 && head_rows % PLAIN_ROW_PAD == 0 && x_step % PLAIN_COL_PAD == 0 && (heads - 1) * (int64_t)x_step + cols <= x_stride && x_stride % 8 == 0,
                "a head's rows are a multiple of %d, its columns start at multiples of %d inside the row", PLAIN_ROW_PAD, PLAIN_COL_PAD);
    TSB_REQUIRE(ctx, y && n_valid > 0 && n_valid <= head_rows && (heads - 1) * (int64_t)y_step + n_valid <= y_stride, "bad output");
    DeviceGuard g(ctx);
    PlainEpi e;
    e.kind = PLAIN_MIXER, e.n_seg = 1;
    PlainSeg& k = e.seg[0];
    k.end = heads * head_rows, k.per = head_rows, k.valid = n_valid, k.step = y_step, k.p = y, k.stride = y_stride;
    k.gate = gate, k.gate_stride = gate_stride, k.gate_step = gate_step;
    PlainMat m{const_cast<void*>(w), (int64_t)heads * head_rows, cols};
    m.group_rows = head_rows, m.group_cols = x_step;
    TSB_CUDA(ctx, launch_plain_gemm(ctx, (cudaStream_t)s, type == TSB_F32, m, x, nullptr, x_stride, x_rows, tokens, e, workspace));
    return TSB_OK;
}

int32_t tsb_post_norm_rows(tsb_ctx* ctx, tsb_stream s, int32_t type, float* x, int32_t d, const float* weight, float eps, int32_t rows, void* out,
                           int64_t out_stride) {
    if (!ctx) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, x && weight && out && d > 0 && rows > 0 && out_stride >= d && (type == TSB_BF16 || type == TSB_F32), "bad arguments");
    TSB_REQUIRE(ctx, (uintptr_t)x % 16 == 0 && (uintptr_t)weight % 16 == 0 && (uintptr_t)out % 16 == 0, "buffers must be 16-byte aligned");
    DeviceGuard g(ctx);
    TSB_CUDA(ctx, launch_post_norm(ctx, (cudaStream_t)s, type == TSB_F32, x, d, weight, eps, rows, out, out_stride));
    return TSB_OK;
}

int32_t tsb_head_norm_rows(tsb_ctx* ctx, tsb_stream s, tsb_kv* cache, int32_t layer, const float* raw, int64_t raw_stride, int32_t n_q, int32_t n_k, int32_t width,
                           const float* q_weight, const float* k_weight, float eps, float temp_coef, int32_t temp_every, const tsb_row_desc* rows_dev,
                           int32_t rows, void* q, int64_t q_stride) {
    if (!ctx || !cache) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, !cache->key_layers.empty() && layer >= 0 && layer < (int)cache->key_layers.size(), "a plain cache and one of its layers expected");
    const KeyView& kv = cache->key_layers[layer];
    TSB_REQUIRE(ctx, raw && rows_dev && rows > 0 && n_q >= 0 && n_k >= 0 && n_k <= kv.kv_heads && n_q + n_k > 0 && width > 0 && width <= kv.head_dim &&
                         raw_stride >= (int64_t)(n_q + n_k) * width && (n_q == 0 || (q && q_weight && q_stride >= (int64_t)n_q * kv.head_dim)) &&
                         (n_k == 0 || k_weight) && temp_every >= 0, "bad arguments");
    DeviceGuard g(ctx);
    HeadNorms h;
    h.raw = raw, h.raw_stride = raw_stride, h.n_q = n_q, h.n_k = n_k, h.width = width, h.q_weight = q_weight, h.k_weight = k_weight, h.eps = eps;
    h.temp_coef = temp_coef, h.temp_every = temp_every, h.q = q, h.q_stride = q_stride, h.q_step = h.q_width = kv.head_dim, h.keys = kv, h.rows = rows_dev;
    TSB_CUDA(ctx, launch_head_norms(ctx, (cudaStream_t)s, kv.elem_bytes == 4, h, rows));
    return TSB_OK;
}

}  // extern "C"
