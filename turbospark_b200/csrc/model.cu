// Sessions and producers: K/V caches and work buffers for a set of independent request streams, the producer calls of
// one stream, speculative rounds and trees over them.  What a model's tensors look like and how its forward pass runs is
// its family's business (ModelFamily in model.cuh: model_blocks.cu, model_rows.cu).
#include <algorithm>
#include <cstring>
#include <memory>
#include <new>
#include <vector>

#include "accept.cuh"
#include "model.cuh"


// ------------------------------------------------------------------ session

int32_t dev_alloc(tsb_ctx* ctx, std::vector<void*>& owned, size_t bytes, void** out) {
    int32_t rc = tsb_alloc(ctx, bytes, out);
    if (rc == TSB_OK) owned.push_back(*out);
    return rc;
}

// One pass through the model's family.  In a replayed round the captured graph already holds this work.
static cudaError_t forward_device(tsb_session* s, ModelRt& rt, const int32_t* tokens_dev, int token_stride,
                                  const tsb_row_desc* rows_dev, int rows, int rows_per_seq, int max_len, LogitRows logits,
                                  int64_t logits_stride, bool last_rows_only = false) {
    if (s->replay) return cudaSuccess;
    Pass p;
    p.tokens = tokens_dev, p.token_stride = token_stride, p.rows_dev = rows_dev, p.rows = rows, p.rows_per_seq = rows_per_seq;
    p.max_len = max_len, p.logits = logits, p.logits_stride = logits_stride, p.last_rows_only = last_rows_only;
    return rt.model->family->forward(s, rt, p);
}

// ------------------------------------------------------------------ model

extern "C" {

void tsb_model_destroy(tsb_model* m) {
    if (!m) return;
    DeviceGuard g(m->ctx);
    cudaDeviceSynchronize();
    m->family->free_tensors(m);
    delete m;
}

int32_t tsb_model_share(tsb_model* dst, int32_t dst_layer, const tsb_model* src, int32_t src_layer) {
    if (!dst || !src) return TSB_ERR_INVALID;
    TSB_REQUIRE(dst->ctx, dst->family == src->family, "models of different families share no tensors");
    return dst->family->share(dst, dst_layer, src, src_layer);
}

int64_t tsb_model_weight_bytes(const tsb_model* m) { return m ? m->family->weight_bytes(m) : 0; }

int32_t tsb_model_logits_f32(const tsb_model* m) { return m && m->family->f32_logits ? 1 : 0; }

}  // extern "C"

// Host side of a forward: descriptors for `n_active` streams x rows_per_seq rows, uploaded through the
// pinned staging ring.  parent == nullptr: a chain.  Returns the device pointers.
int32_t stage_rows(tsb_session* s, ModelRt& rt, const int32_t* streams, int n_active, int rows_per_seq,
                          const int32_t* slot_parent, const int32_t* tokens_host /* may be null */,
                          const tsb_row_desc** rows_dev, const int32_t** tokens_dev, int* max_len) {
    tsb_ctx* ctx = s->ctx;
    const int rows = n_active * rows_per_seq;
    TSB_REQUIRE(ctx, rows <= s->n_streams * s->max_rows, "%d rows exceed the session's %d", rows, s->n_streams * s->max_rows);
    TSB_REQUIRE(ctx, rows_per_seq <= 128, "at most 128 in-flight rows per stream");
    bool chain = true;
    for (int j = 0; slot_parent && j < rows_per_seq; j++) chain &= slot_parent[j] == j - 1;
    if (!chain && !rt.model->family->trees)
        return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "%s models verify chains only: a row's state is its predecessor's, not its parent's", rt.model->family->name);
    if (s->stage_used + rows > s->stage_cap) {
        if (s->replay || s->capturing) return tsb_fail(ctx, TSB_ERR_STATE, "staging ring overflow inside a captured round");
        // the ring is reused only after the work that read it has finished
        TSB_CUDA(ctx, cudaStreamSynchronize(s->stream));
        s->stage_used = 0;
    }
    tsb_row_desc* hd = s->stage_rows_host + s->stage_used;
    int32_t* ht = s->stage_tok_host + s->stage_used;
    std::vector<int> depth(rows_per_seq, 0);
    std::vector<uint64_t> mlo(rows_per_seq, 0), mhi(rows_per_seq, 0);
    for (int j = 0; j < rows_per_seq; j++) {
        if (slot_parent) {
            if (j == 0) {
                TSB_REQUIRE(ctx, slot_parent[0] == -1, "a tree's slot 0 is the anchor (parent -1)");
            } else {
                const int p = slot_parent[j];
                TSB_REQUIRE(ctx, p >= 0 && p < j, "slot %d's parent %d must precede it", j, p);
                depth[j] = depth[p] + 1;
                mlo[j] = mlo[p], mhi[j] = mhi[p];
            }
        } else {
            depth[j] = j;
            if (j) mlo[j] = mlo[j - 1], mhi[j] = mhi[j - 1];
        }
        if (j < 64) mlo[j] |= 1ull << j; else mhi[j] |= 1ull << (j - 64);
    }
    int ml = 0;
    for (int a = 0; a < n_active; a++) {
        const int seq = streams[a];
        TSB_REQUIRE(ctx, seq >= 0 && seq < s->n_streams, "stream %d outside the session", seq);
        const int64_t base = tsb_kv_cursor(rt.kv, seq);
        if (base + rows_per_seq > rt.model->cfg.max_context)
            return tsb_fail(ctx, TSB_ERR_STATE, "stream %d: %lld + %d rows exceed the context window %d", seq, (long long)base,
                            rows_per_seq, rt.model->cfg.max_context);
        int32_t rc = tsb_kv_reserve(rt.kv, seq, base + rows_per_seq);
        if (rc) return rc;
        for (int j = 0; j < rows_per_seq; j++) {
            tsb_row_desc& d = hd[a * rows_per_seq + j];
            d.seq = seq, d.base = (int32_t)base, d.slot = j, d.position = (int32_t)base + depth[j];
            d.mask[0] = mlo[j], d.mask[1] = mhi[j];
            if (tokens_host) ht[a * rows_per_seq + j] = tokens_host[a * rows_per_seq + j];
        }
        ml = ml > (int)base + rows_per_seq ? ml : (int)base + rows_per_seq;
    }
    tsb_row_desc* dd = s->stage_rows_dev + s->stage_used;
    int32_t* dt = s->stage_tok_dev + s->stage_used;
    if (!s->replay) {
        TSB_CUDA(ctx, cudaMemcpyAsync(dd, hd, rows * sizeof(tsb_row_desc), cudaMemcpyHostToDevice, s->stream));
        if (tokens_host) TSB_CUDA(ctx, cudaMemcpyAsync(dt, ht, rows * sizeof(int32_t), cudaMemcpyHostToDevice, s->stream));
    }
    s->stage_used += rows;
    *rows_dev = dd;
    if (tokens_dev) *tokens_dev = dt;
    *max_len = ml;
    return TSB_OK;
}

extern "C" {
static int32_t drafter_catch_up(tsb_session* s, int stream, int64_t upto);
}

// forward + cursor advance for one stream (the single-stream producer calls)
static int32_t forward_stream(tsb_session* s, ModelRt& rt, int stream, const int32_t* tokens, int n, const int32_t* slot_parent,
                              LogitRows logits_dev, void* logits_out_host) {
    tsb_ctx* ctx = s->ctx;
    const tsb_row_desc* rd;
    const int32_t* td;
    int max_len;
    int32_t rc = stage_rows(s, rt, &stream, 1, n, slot_parent, tokens, &rd, &td, &max_len);
    if (rc) return rc;
    const int vocab = rt.model->cfg.vocab;
    TSB_CUDA(ctx, forward_device(s, rt, td, 1, rd, n, n, max_len, logits_dev, vocab));
    tsb_kv_set_cursor(rt.kv, stream, tsb_kv_cursor(rt.kv, stream) + n);
    if (logits_dev && logits_out_host)
        TSB_CUDA(ctx, cudaMemcpyAsync(logits_out_host, logits_dev.p, (size_t)n * vocab * logits_dev.bytes(), cudaMemcpyDeviceToHost, s->stream));
    if (logits_out_host) return tsb_stream_sync(ctx, s->stream);
    return TSB_OK;
}

extern "C" {

int32_t tsb_session_create(tsb_ctx* ctx, const tsb_model* target, const tsb_model* draft, int32_t n_streams,
                           int32_t max_rows, int32_t page_tokens, tsb_session** out) {
    return tsb_session_create_pool(ctx, target, draft, n_streams, max_rows, page_tokens, 0, 0, out);
}

int32_t tsb_session_create_pool(tsb_ctx* ctx, const tsb_model* target, const tsb_model* draft, int32_t n_streams, int32_t max_rows,
                                int32_t page_tokens, int64_t pool_tokens, int32_t step_rows, tsb_session** out) {
    if (!ctx || !target || !out) return TSB_ERR_INVALID;
    *out = nullptr;
    TSB_REQUIRE(ctx, pool_tokens >= 0 && step_rows >= 0 && page_tokens > 0, "bad pool or step size");
    TSB_REQUIRE(ctx, n_streams > 0 && max_rows > 0 && max_rows <= 128, "n_streams must be positive and max_rows in 1..128");
    int32_t rc = target->family->complete(target);
    if (rc) return rc;
    TSB_REQUIRE(ctx, step_rows == 0 || target->family->ragged, "%s models take no mixed steps", target->family->name);
    if (draft) {
        if ((rc = draft->family->complete(draft))) return rc;
        TSB_REQUIRE(ctx, draft->family->f32_logits == target->family->f32_logits, "target and drafter write logits of different types");
        TSB_REQUIRE(ctx, draft->cfg.vocab == target->cfg.vocab, "the drafter must share the target's vocabulary");
    }
    if (target->cfg.vocab > accept_max_vocab())
        return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "vocabulary %d exceeds the device sampler's %d", target->cfg.vocab, accept_max_vocab());
    DeviceGuard g(ctx);
    tsb_session* s = new (std::nothrow) tsb_session();
    if (!s) return TSB_ERR_OOM;
    s->ctx = ctx, s->n_streams = n_streams, s->max_rows = max_rows;
    s->generated.assign(n_streams, 0);
    auto fail = [&](int32_t code) {
        tsb_session_destroy(s);
        return code;
    };
    if (cudaStreamCreateWithFlags(&s->stream, cudaStreamNonBlocking) != cudaSuccess) return fail(TSB_ERR_CUDA);
    for (auto& ev : s->ev)
        if (cudaEventCreate(&ev) != cudaSuccess) return fail(TSB_ERR_CUDA);
    s->pass_rows = std::max(n_streams * max_rows, step_rows);
    s->logits_f32 = target->family->f32_logits;
    // pool_tokens == 0: every stream can reach the context window; otherwise the streams share that many positions' pages
    auto shape_of = [&](const tsb_model* m, bool is_draft) {
        SessionShape sh;
        sh.n_streams = n_streams, sh.max_rows = max_rows, sh.page_tokens = page_tokens;
        sh.pages_per_seq = (m->cfg.max_context + page_tokens - 1) / page_tokens;
        sh.num_pages = pool_tokens > 0 ? (int)((pool_tokens + page_tokens - 1) / page_tokens) : sh.pages_per_seq * n_streams;
        sh.pass_rows = is_draft ? n_streams * max_rows : s->pass_rows;
        return sh;
    };
    if ((rc = target->family->runtime_init(s, s->target, target, shape_of(target, false), false))) return fail(rc);
    if (draft && (rc = draft->family->runtime_init(s, s->draft, draft, shape_of(draft, true), true))) return fail(rc);
    s->has_draft = draft != nullptr;
    {
        const char* env = getenv("TSB_GRAPH");
        if (env && env[0] == '0') s->use_graph = false;
    }
    const int R = n_streams * max_rows, V = target->cfg.vocab;
    auto A = [&](size_t bytes, void** p) { return dev_alloc(ctx, s->owned, bytes, p); };
    s->logits_target.f32 = s->logits_draft.f32 = s->logits_f32;
    const size_t lb = s->logits_f32 ? 4 : 2;
    s->logit_rows = std::max(R, std::min(s->pass_rows, 256));
    if ((rc = A((size_t)s->logit_rows * V * lb, &s->logits_target.p))) return fail(rc);
    if (draft && (rc = A((size_t)R * V * lb, &s->logits_draft.p))) return fail(rc);
    if ((rc = A((size_t)(R + 2 * n_streams) * sizeof(int32_t), (void**)&s->feed_dev))) return fail(rc);
    s->pair_dev = s->feed_dev + R;
    if ((rc = A((size_t)n_streams * (3 * max_rows + 2) * sizeof(uint64_t), (void**)&s->uniforms_dev))) return fail(rc);
    if ((rc = A((size_t)n_streams * sizeof(tsb_accept_out), (void**)&s->accept_out_dev))) return fail(rc);
    s->accept_scratch_bytes = accept_scratch_bytes(n_streams, max_rows, V);
    if ((rc = A(s->accept_scratch_bytes, &s->accept_scratch))) return fail(rc);
    if ((rc = A((size_t)n_streams * sizeof(int32_t), (void**)&s->tok1_dev))) return fail(rc);
    if ((rc = A((size_t)128 * 9 * sizeof(int32_t), (void**)&s->tree_dev))) return fail(rc);
    // pinned staging: descriptors and tokens of several forwards in flight
    s->stage_cap = std::max(R * (2 * max_rows + 8), 2 * s->pass_rows);
    if (cudaMallocHost((void**)&s->stage_rows_host, (size_t)s->stage_cap * sizeof(tsb_row_desc)) != cudaSuccess) return fail(TSB_ERR_CUDA);
    if (cudaMallocHost((void**)&s->stage_tok_host, (size_t)s->stage_cap * sizeof(int32_t)) != cudaSuccess) return fail(TSB_ERR_CUDA);
    if ((rc = A((size_t)s->stage_cap * sizeof(tsb_row_desc), (void**)&s->stage_rows_dev))) return fail(rc);
    if ((rc = A((size_t)s->stage_cap * sizeof(int32_t), (void**)&s->stage_tok_dev))) return fail(rc);
    if (target->family->ragged) {
        s->stage_int_cap = std::max(64 * s->pass_rows, 4096);
        if (cudaMallocHost((void**)&s->stage_int_host, (size_t)s->stage_int_cap * sizeof(int32_t)) != cudaSuccess) return fail(TSB_ERR_CUDA);
        if ((rc = A((size_t)s->stage_int_cap * sizeof(int32_t), (void**)&s->stage_int_dev))) return fail(rc);
    }
    if (cudaMallocHost((void**)&s->accept_out_host, (size_t)n_streams * sizeof(tsb_accept_out)) != cudaSuccess) return fail(TSB_ERR_CUDA);
    if (cudaMallocHost((void**)&s->uniforms_host, (size_t)n_streams * (3 * max_rows + 2) * sizeof(uint64_t)) != cudaSuccess) return fail(TSB_ERR_CUDA);
    if (cudaMallocHost((void**)&s->feed_host, (size_t)(R + 2 * n_streams) * sizeof(int32_t)) != cudaSuccess) return fail(TSB_ERR_CUDA);
    s->pair_host = s->feed_host + R;
    if (cudaMallocHost((void**)&s->logits_host, (size_t)V * lb) != cudaSuccess) return fail(TSB_ERR_CUDA);
    *out = s;
    return TSB_OK;
}

void tsb_session_destroy(tsb_session* s) {
    if (!s) return;
    DeviceGuard g(s->ctx);
    cudaDeviceSynchronize();
    if (s->graph) cudaGraphExecDestroy(s->graph);
    for (ModelRt* rt : {&s->target, &s->draft})
        if (rt->model && rt->model->family->runtime_free) rt->model->family->runtime_free(*rt);
    for (void* p : s->owned) tsb_free(s->ctx, p);
    if (s->target.kv) tsb_kv_destroy(s->target.kv);
    if (s->draft.kv) tsb_kv_destroy(s->draft.kv);
    cudaFreeHost(s->stage_rows_host), cudaFreeHost(s->stage_tok_host), cudaFreeHost(s->accept_out_host);
    cudaFreeHost(s->uniforms_host), cudaFreeHost(s->feed_host), cudaFreeHost(s->logits_host), cudaFreeHost(s->stage_int_host);
    for (auto& ev : s->ev)
        if (ev) cudaEventDestroy(ev);
    if (s->stream) cudaStreamDestroy(s->stream);
    delete s;
}

int32_t tsb_session_set_comm(tsb_session* s, tsb_comm* c) {
    if (!s) return TSB_ERR_INVALID;
    DeviceGuard g(s->ctx);
    TSB_CUDA(s->ctx, cudaStreamSynchronize(s->stream));
    if (s->graph) cudaGraphExecDestroy(s->graph), s->graph = nullptr;  // captured rounds hold the old exchange steps
    s->comm = c;
    return TSB_OK;
}

tsb_kv* tsb_session_kv(tsb_session* s, int32_t which) { return !s ? nullptr : (which == 0 ? s->target.kv : s->draft.kv); }

// ---- LogitProducer / SpeculativeProducer, one stream ----------------------

int32_t tsb_producer_reset(tsb_session* s, int32_t stream) {
    if (!s) return TSB_ERR_INVALID;
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    DeviceGuard g(s->ctx);
    TSB_CUDA(s->ctx, cudaStreamSynchronize(s->stream));
    int32_t rc = tsb_kv_reset(s->target.kv, stream);
    if (rc) return rc;
    s->target.fed[stream].clear();
    s->target.pending[stream] = PendingVerify();
    s->generated[stream] = 0;
    if (s->has_draft) {
        if ((rc = tsb_kv_reset(s->draft.kv, stream))) return rc;
    }
    return TSB_OK;
}

int32_t tsb_session_set_generated(tsb_session* s, int32_t stream, int32_t generated) {
    if (!s) return TSB_ERR_INVALID;
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams && generated >= 0, "bad stream or count");
    s->generated[stream] = generated;
    return TSB_OK;
}

static int32_t check_position(tsb_session* s, ModelRt& rt, int stream, int64_t position) {
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    const int64_t cur = tsb_kv_cursor(rt.kv, stream);
    if (position != cur)  // crates/runtime/src/families/qwen/batched.rs:150-160: start must equal the cursor
        return tsb_fail(s->ctx, TSB_ERR_STATE, "position %lld does not continue the cache (cursor %lld)", (long long)position,
                        (long long)cur);
    return TSB_OK;
}

static void record_fed(ModelRt& rt, int stream, int64_t position, const int32_t* tokens, int n) {
    auto& f = rt.fed[stream];
    f.resize((size_t)position);
    f.insert(f.end(), tokens, tokens + n);
}

int32_t tsb_producer_produce(tsb_session* s, int32_t stream, int32_t token, int64_t position, void* logits_out_host) {
    if (!s) return TSB_ERR_INVALID;
    DeviceGuard g(s->ctx);
    int32_t rc = check_position(s, s->target, stream, position);
    if (rc) return rc;
    record_fed(s->target, stream, position, &token, 1);
    return forward_stream(s, s->target, stream, &token, 1, nullptr, s->logits_target, logits_out_host);
}

int32_t tsb_producer_produce_prefill(tsb_session* s, int32_t stream, int32_t token, int64_t position) {
    if (!s) return TSB_ERR_INVALID;
    DeviceGuard g(s->ctx);
    int32_t rc = check_position(s, s->target, stream, position);
    if (rc) return rc;
    record_fed(s->target, stream, position, &token, 1);
    return forward_stream(s, s->target, stream, &token, 1, nullptr, LogitRows(), nullptr);
}

// the drafter is a stand-alone decoder: bring its cache up to `upto` from the record of fed tokens
static int32_t drafter_catch_up(tsb_session* s, int stream, int64_t upto) {
    ModelRt& d = s->draft;
    const auto& fed = s->target.fed[stream];
    while (tsb_kv_cursor(d.kv, stream) < upto) {
        const int64_t p = tsb_kv_cursor(d.kv, stream);
        if ((size_t)p >= fed.size()) return tsb_fail(s->ctx, TSB_ERR_STATE, "drafter position %lld was never fed to the target", (long long)p);
        int64_t n64 = upto - p;
        if (n64 > s->max_rows) n64 = s->max_rows;
        if (n64 > (int64_t)fed.size() - p) n64 = (int64_t)fed.size() - p;
        const int n = (int)n64;
        int32_t rc = forward_stream(s, d, stream, fed.data() + p, n, nullptr, LogitRows(), nullptr);
        if (rc) return rc;
    }
    return TSB_OK;
}

static int32_t drafter_step(tsb_session* s, int32_t stream, int32_t next, int64_t position, bool head, void* logits_out_host) {
    if (!s) return TSB_ERR_INVALID;
    if (!s->has_draft) return tsb_fail(s->ctx, TSB_ERR_STATE, "the session has no drafter");
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    DeviceGuard g(s->ctx);
    int32_t rc = drafter_catch_up(s, stream, position + 1);
    if (rc) return rc;
    if ((rc = check_position(s, s->draft, stream, position + 1))) return rc;
    return forward_stream(s, s->draft, stream, &next, 1, nullptr, head ? s->logits_draft : LogitRows(), logits_out_host);
}

int32_t tsb_producer_prime_drafter(tsb_session* s, int32_t stream, int32_t next, int64_t position) {
    return drafter_step(s, stream, next, position, false, nullptr);
}
int32_t tsb_producer_draft_step(tsb_session* s, int32_t stream, int32_t next, int64_t position, void* logits_out_host) {
    return drafter_step(s, stream, next, position, true, logits_out_host);
}

int32_t tsb_producer_verify(tsb_session* s, int32_t stream, const int32_t* feed, int32_t n, int64_t base, void* logits_out_host) {
    if (!s) return TSB_ERR_INVALID;
    TSB_REQUIRE(s->ctx, feed && n > 0 && n <= s->max_rows, "verify takes 1..%d rows", s->max_rows);
    DeviceGuard g(s->ctx);
    int32_t rc = check_position(s, s->target, stream, base);
    if (rc) return rc;
    record_fed(s->target, stream, base, feed, n);
    PendingVerify& pv = s->target.pending[stream];
    pv.active = true, pv.tree = false, pv.base = base, pv.rows = n, pv.feed.clear(), pv.drafter_rows = 0;
    return forward_stream(s, s->target, stream, feed, n, nullptr, s->logits_target, logits_out_host);
}

int32_t tsb_producer_verify_tree(tsb_session* s, int32_t stream, const int32_t* feed, const int32_t* slot_parent, int32_t n,
                                 int64_t base, void* logits_out_host) {
    if (!s) return TSB_ERR_INVALID;
    TSB_REQUIRE(s->ctx, feed && slot_parent && n > 0 && n <= s->max_rows, "verify_tree takes 1..%d rows", s->max_rows);
    DeviceGuard g(s->ctx);
    int32_t rc = check_position(s, s->target, stream, base);
    if (rc) return rc;
    // the slots' tokens are kept until compact_tree says which of them form the accepted path
    PendingVerify& pv = s->target.pending[stream];
    const int drafted = pv.active && pv.tree && pv.base == base && pv.rows == 0 ? pv.drafter_rows : 0;  // left by draft_tree
    pv.active = true, pv.tree = true, pv.base = base, pv.rows = n, pv.feed.assign(feed, feed + n), pv.drafter_rows = drafted;
    return forward_stream(s, s->target, stream, feed, n, slot_parent, s->logits_target, logits_out_host);
}

int32_t tsb_session_verify_tree(tsb_session* s, const int32_t* feed, const int32_t* slot_parent, int32_t n, void* logits_out_host) {
    if (!s) return TSB_ERR_INVALID;
    tsb_ctx* ctx = s->ctx;
    TSB_REQUIRE(ctx, feed && slot_parent && n > 0 && n <= s->max_rows, "verify_tree takes 1..%d rows per stream", s->max_rows);
    DeviceGuard g(ctx);
    const int S = s->n_streams;
    std::vector<int32_t> streams(S);
    for (int b = 0; b < S; b++) streams[b] = b;
    const tsb_row_desc* rd;
    const int32_t* td;
    int max_len;
    int32_t rc = stage_rows(s, s->target, streams.data(), S, n, slot_parent, feed, &rd, &td, &max_len);
    if (rc) return rc;
    const int vocab = s->target.model->cfg.vocab;
    TSB_CUDA(ctx, forward_device(s, s->target, td, 1, rd, S * n, n, max_len, s->logits_target, vocab));
    for (int b = 0; b < S; b++) {
        const int64_t base = tsb_kv_cursor(s->target.kv, b);
        PendingVerify& pv = s->target.pending[b];
        pv.active = true, pv.tree = true, pv.base = base, pv.rows = n, pv.feed.assign(feed + (size_t)b * n, feed + (size_t)(b + 1) * n), pv.drafter_rows = 0;
        tsb_kv_set_cursor(s->target.kv, b, base + n);
    }
    if (logits_out_host) {
        TSB_CUDA(ctx, cudaMemcpyAsync(logits_out_host, s->logits_target.p, (size_t)S * n * vocab * s->logits_target.bytes(), cudaMemcpyDeviceToHost, s->stream));
        return tsb_stream_sync(ctx, s->stream);
    }
    return TSB_OK;
}

int32_t tsb_producer_compact_tree(tsb_session* s, int32_t stream, int64_t base, const uint32_t* path, int32_t keep) {
    if (!s) return TSB_ERR_INVALID;
    tsb_ctx* ctx = s->ctx;
    TSB_REQUIRE(ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    PendingVerify& pv = s->target.pending[stream];
    if (!pv.active || !pv.tree || pv.base != base)
        return tsb_fail(ctx, TSB_ERR_STATE, "compact_tree at %lld has no tree verify to compact", (long long)base);
    TSB_REQUIRE(ctx, path && keep >= 1 && keep <= pv.rows && path[0] == 0, "the path starts at slot 0 and has 1..%d entries", pv.rows);
    for (int r = 1; r < keep; r++) TSB_REQUIRE(ctx, path[r] > path[r - 1] && (int)path[r] < pv.rows, "path entries increase and stay inside the verify");
    DeviceGuard g(ctx);
    int32_t rc = tsb_kv_commit_path(ctx, s->stream, s->target.kv, stream, base, path, keep);
    if (rc) return rc;
    // the drafter holds rows only for the slots it was run over: the part of the path it has is compacted too, the
    // rest is replayed from the record of fed tokens before its next step
    int dkeep = 0;
    if (s->has_draft && pv.drafter_rows > 0 && tsb_kv_cursor(s->draft.kv, stream) == base) {
        while (dkeep < keep && (int)path[dkeep] < pv.drafter_rows) dkeep++;
        if (dkeep > 0 && (rc = tsb_kv_commit_path(ctx, s->stream, s->draft.kv, stream, base, path, dkeep))) return rc;
    }
    if ((rc = tsb_stream_sync(ctx, s->stream))) return rc;
    // the verify left the cursor past every slot; the kept rows now sit at base .. base + keep
    if (dkeep > 0) tsb_kv_set_cursor(s->draft.kv, stream, base + dkeep);
    auto& fed = s->target.fed[stream];
    if ((int64_t)fed.size() < base) return tsb_fail(ctx, TSB_ERR_STATE, "the record of fed tokens ends before %lld", (long long)base);
    fed.resize((size_t)base);
    for (int r = 0; r < keep; r++) fed.push_back(pv.feed[path[r]]);
    // the slots past the path are dropped from the record; their cache rows are cut by rollback_retaining
    pv.tree = false, pv.feed.clear();  // compacted: what remains pending is a chain of pv.rows rows, of which `keep` matter
    return TSB_OK;
}

int64_t tsb_producer_checkpoint(tsb_session* s, int32_t stream) { return s ? tsb_kv_cursor(s->target.kv, stream) : -1; }

int32_t tsb_producer_rollback(tsb_session* s, int32_t stream, int64_t point) {
    return tsb_producer_rollback_retaining(s, stream, point, 0);
}

// crates/runtime/src/real_forward_rollback.rs:268-405 for a pure-attention model: a cursor move.
int32_t tsb_producer_rollback_retaining(tsb_session* s, int32_t stream, int64_t point, int32_t keep_rows) {
    if (!s) return TSB_ERR_INVALID;
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    const int64_t cur = tsb_kv_cursor(s->target.kv, stream);
    if (point < 0 || keep_rows < 0 || point + keep_rows > cur)
        return tsb_fail(s->ctx, TSB_ERR_STATE, "cannot keep %d rows after %lld: the cursor is %lld", keep_rows, (long long)point,
                        (long long)cur);
    // the record of fed tokens is only ever cut here: rows nobody recorded cannot be kept
    if ((int64_t)s->target.fed[stream].size() < point + keep_rows)
        return tsb_fail(s->ctx, TSB_ERR_STATE, "the record of fed tokens holds %zu entries, fewer than the %lld rows to keep "
                        "(after verify_tree, compact_tree comes first)", s->target.fed[stream].size(), (long long)(point + keep_rows));
    int32_t rc = tsb_kv_set_cursor(s->target.kv, stream, point + keep_rows);
    if (rc) return rc;
    s->target.fed[stream].resize((size_t)(point + keep_rows));
    return TSB_OK;
}

int32_t tsb_producer_commit_pending(tsb_session* s, int32_t stream, int32_t keep_rows) {
    if (!s) return TSB_ERR_INVALID;
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    PendingVerify& pv = s->target.pending[stream];
    if (!pv.active) return TSB_OK;
    if (keep_rows < 0 || keep_rows > pv.rows)
        return tsb_fail(s->ctx, TSB_ERR_STATE, "commit_pending(%d): the last verify fed %d rows", keep_rows, pv.rows);
    pv = PendingVerify();
    return TSB_OK;
}

int32_t tsb_producer_discard_pending(tsb_session* s, int32_t stream) {
    if (!s) return TSB_ERR_INVALID;
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    PendingVerify& pv = s->target.pending[stream];
    if (!pv.active) return TSB_OK;
    DeviceGuard g(s->ctx);
    cudaStreamSynchronize(s->stream);  // whatever the failed round enqueued is over before the cursors move
    const int64_t base = pv.base;
    pv = PendingVerify();
    if (tsb_kv_cursor(s->target.kv, stream) > base) tsb_kv_set_cursor(s->target.kv, stream, base);
    if (s->target.fed[stream].size() > (size_t)base) s->target.fed[stream].resize((size_t)base);
    if (s->has_draft && tsb_kv_cursor(s->draft.kv, stream) > base + 1) tsb_kv_set_cursor(s->draft.kv, stream, base + 1);
    return TSB_OK;
}

int32_t tsb_producer_supports_retaining_rollback(const tsb_session* s) { return s ? 1 : 0; }
int32_t tsb_producer_supports_headless_prefill(const tsb_session* s) { return s ? 1 : 0; }
int32_t tsb_producer_drafts_block_passes(const tsb_session* s) {
    (void)s;
    return 0;
}

int32_t tsb_session_set_tree(tsb_session* s, int32_t nodes, int32_t levels, const int32_t* branching, int32_t best_first, int32_t cand) {
    if (!s) return TSB_ERR_INVALID;
    tsb_ctx* ctx = s->ctx;
    TreeShape t;
    if (nodes == 0) {
        s->tree = t;
        return TSB_OK;
    }
    TSB_REQUIRE(ctx, nodes >= 1 && nodes + 1 <= s->max_rows && nodes + 1 <= 128, "a tree of %d nodes plus the anchor exceeds the session's %d rows", nodes, s->max_rows);
    TSB_REQUIRE(ctx, levels >= 1 && levels <= 8, "levels must be 1..8");
    t.nodes = nodes, t.levels = levels, t.best_first = best_first ? 1 : 0, t.cand = cand;
    if (best_first) {
        TSB_REQUIRE(ctx, cand >= 1 && cand <= 8, "cand must be 1..8");
    } else {
        TSB_REQUIRE(ctx, branching != nullptr, "a static tree needs its branching list");
        for (int l = 0; l < levels; l++) {
            TSB_REQUIRE(ctx, branching[l] >= 1 && branching[l] <= 8, "branching must be 1..8");
            t.branching[l] = branching[l];
        }
    }
    s->tree = t;
    return TSB_OK;
}

int32_t tsb_producer_tree_nodes(const tsb_session* s) { return s ? s->tree.nodes : 0; }

int32_t tsb_tree_slot_parents(const tsb_tree_node* tree, int32_t n, int32_t* out) {
    if ((!tree && n) || !out || n < 0) return TSB_ERR_INVALID;
    out[0] = -1;
    for (int i = 0; i < n; i++) out[i + 1] = tree[i].parent < 0 ? 0 : tree[i].parent + 1;
    return TSB_OK;
}

int32_t tsb_best_first_tree(const float* scores, int32_t depth_max, int32_t branch, int32_t nodes, tsb_tree_node* out) {
    if (!scores || !out || branch <= 0) return 0;
    std::vector<tsb_tree_node> t;
    best_first_tree(depth_max, nodes, branch,
                    [&](int depth, int /*parent*/, float* sc) -> int32_t {
                        for (int c = 0; c < branch; c++) sc[c] = scores[(size_t)depth * branch + c];
                        return 0;
                    },
                    t);
    std::copy(t.begin(), t.end(), out);
    return (int32_t)t.size();
}

int32_t tsb_tree_accept(const tsb_tree_node* tree, const int32_t* tokens, int32_t n, const int32_t* target_pick, int32_t* accepted_out) {
    if ((!tree && n) || (!tokens && n) || !target_pick || !accepted_out || n < 0) return 0;
    int at = -1, k = 0;
    for (;;) {
        const int32_t want = target_pick[at + 1];
        int hit = -1;
        for (int id = 0; id < n && hit < 0; id++)
            if (tree[id].parent == at && tokens[id] == want) hit = id;
        if (hit < 0) return k;
        accepted_out[k++] = hit;
        at = hit;
    }
}

int32_t tsb_producer_draft_tree(tsb_session* s, int32_t stream, int32_t anchor, int64_t base, int32_t nodes, tsb_tree_node* tree_out,
                                int32_t* tokens_out, int32_t* n_out) {
    if (!s || !tree_out || !tokens_out || !n_out) return TSB_ERR_INVALID;
    tsb_ctx* ctx = s->ctx;
    TSB_REQUIRE(ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    if (s->tree.nodes == 0) return tsb_fail(ctx, TSB_ERR_STATE, "this producer verifies chains only (tsb_session_set_tree turns trees on)");
    TSB_REQUIRE(ctx, nodes >= 1 && nodes <= s->tree.nodes, "nodes must be 1..%d", s->tree.nodes);
    DeviceGuard g(ctx);
    TreeShape shape = s->tree;
    shape.nodes = nodes;
    std::vector<int32_t> feed, parent;
    std::vector<tsb_tree_node> tree;
    int drafter_rows = 0;
    int32_t rc = session_draft_tree(s, stream, shape, anchor, base, feed, parent, tree, &drafter_rows);
    if (rc) return rc;
    for (size_t i = 0; i < tree.size(); i++) tree_out[i] = tree[i], tokens_out[i] = feed[i + 1];
    *n_out = (int32_t)tree.size();
    // remembered for the verify_tree / compact_tree that follow: which slots the drafter's cache holds
    PendingVerify& pv = s->target.pending[stream];
    pv = PendingVerify();
    pv.active = true, pv.tree = true, pv.base = base, pv.rows = 0, pv.drafter_rows = drafter_rows;
    return TSB_OK;
}

int32_t tsb_producer_draft_block(tsb_session* s, int32_t stream, int32_t anchor, int64_t base, int32_t block, int32_t* proposals_out) {
    if (!s || !proposals_out) return TSB_ERR_INVALID;
    tsb_ctx* ctx = s->ctx;
    if (!s->has_draft) return tsb_fail(ctx, TSB_ERR_STATE, "the session has no drafter");
    TSB_REQUIRE(ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    TSB_REQUIRE(ctx, block >= 1 && block <= 15, "block must be 1..=15");
    DeviceGuard g(ctx);
    const int V = s->draft.model->cfg.vocab;
    int32_t tok = anchor;
    for (int i = 0; i <= block; i++) {
        // step i feeds the token at base + i; its logits give proposal i (the last step is taken for its row alone)
        int32_t rc = drafter_step(s, stream, tok, base + i - 1, i < block, nullptr);
        if (rc) return rc;
        if (i == block) break;
        TSB_CUDA(ctx, launch_argmax_rows(ctx, s->stream, s->logits_draft, 1, V, s->accept_scratch));
        std::vector<uint8_t> stats(accept_row_stats_bytes());
        TSB_CUDA(ctx, cudaMemcpyAsync(stats.data(), s->accept_scratch, stats.size(), cudaMemcpyDeviceToHost, s->stream));
        if ((rc = tsb_stream_sync(ctx, s->stream))) return rc;
        int32_t am, bad;
        accept_row_stats_read(stats.data(), 0, &am, &bad);
        if (bad) return tsb_fail(ctx, TSB_ERR_DEVICE, "the drafter's logits at step %d are not finite", i);
        proposals_out[i] = tok = am;
    }
    return TSB_OK;
}

int32_t tsb_producer_rewind_drafter(tsb_session* s, int32_t stream, int64_t position) {
    if (!s) return TSB_ERR_INVALID;
    if (!s->has_draft) return TSB_OK;
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    if (tsb_kv_cursor(s->draft.kv, stream) > position + 1) return tsb_kv_set_cursor(s->draft.kv, stream, position + 1);
    return TSB_OK;
}

int64_t tsb_producer_try_reuse_prefix(tsb_session* s, int32_t stream, const int32_t* prompt_ids, int32_t n) {
    if (!s || !prompt_ids || n <= 0 || stream < 0 || stream >= s->n_streams) return 0;
    auto& fed = s->target.fed[stream];
    const int64_t cur = tsb_kv_cursor(s->target.kv, stream);
    int64_t lim = std::min<int64_t>(std::min<int64_t>(cur, (int64_t)fed.size()), (int64_t)n - 1);
    int64_t keep = 0;
    while (keep < lim && fed[(size_t)keep] == prompt_ids[keep]) keep++;
    if (tsb_kv_set_cursor(s->target.kv, stream, keep) != TSB_OK) {  // a state that no longer reaches back that far: start over
        keep = 0;
        tsb_kv_set_cursor(s->target.kv, stream, 0);
    }
    fed.resize((size_t)keep);
    if (s->has_draft && tsb_kv_cursor(s->draft.kv, stream) > keep && tsb_kv_set_cursor(s->draft.kv, stream, keep) != TSB_OK)
        tsb_kv_set_cursor(s->draft.kv, stream, 0);
    return keep;
}

int32_t tsb_producer_record_committed(tsb_session* s, int32_t stream, const int32_t* tokens, int32_t n, int64_t pos0) {
    if (!s || (!tokens && n) || n < 0) return TSB_ERR_INVALID;
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    TSB_REQUIRE(s->ctx, pos0 >= 0 && pos0 <= (int64_t)s->target.fed[stream].size(), "pos0 %lld does not continue the record", (long long)pos0);
    record_fed(s->target, stream, pos0, tokens, n);
    return TSB_OK;
}

// ---- one lockstep round over every stream ----------------------------------

int32_t tsb_session_fill_context(tsb_session* s, int64_t tokens, uint64_t seed) {
    if (!s) return TSB_ERR_INVALID;
    DeviceGuard g(s->ctx);
    for (int q = 0; q < s->n_streams; q++) {
        int32_t rc = s->target.model->family->fill_context(s, s->target, q, tokens, seed + 2 * q);
        if (rc) return rc;
        tsb_kv_set_cursor(s->target.kv, q, tokens);
        s->target.fed[q].assign((size_t)tokens, 0);
        if (s->has_draft) {
            if ((rc = s->draft.model->family->fill_context(s, s->draft, q, tokens, seed + 2 * q + 1))) return rc;
            tsb_kv_set_cursor(s->draft.kv, q, tokens);
        }
    }
    return tsb_stream_sync(s->ctx, s->stream);
}

}  // extern "C"

int32_t session_stage_history(tsb_session* s, const int32_t* streams, int n_active, const int32_t* next_tokens) {
    tsb_ctx* ctx = s->ctx;
    const int max_ctx = s->target.model->cfg.max_context, V = s->target.model->cfg.vocab;
    if (!s->hist_dev) {
        TSB_CUDA(ctx, cudaMalloc((void**)&s->hist_dev, (size_t)s->n_streams * max_ctx * sizeof(int32_t)));
        s->owned.push_back(s->hist_dev);
        TSB_CUDA(ctx, cudaMalloc((void**)&s->hist_len_dev, (size_t)s->n_streams * 2 * sizeof(int32_t)));
        s->owned.push_back(s->hist_len_dev);
        s->gen_dev = s->hist_len_dev + s->n_streams;
        TSB_CUDA(ctx, cudaMalloc(&s->pen_scratch, accept_history_scratch_bytes(s->n_streams, std::min(15, s->max_rows - 1 > 0 ? s->max_rows - 1 : 1), V)));
        s->owned.push_back(s->pen_scratch);
    }
    s->hist_host.assign((size_t)n_active * max_ctx + 2 * (size_t)n_active, 0);
    int32_t* lens = s->hist_host.data() + (size_t)n_active * max_ctx;
    for (int a = 0; a < n_active; a++) {
        const int q = streams[a];
        const auto& fed = s->target.fed[q];
        const int64_t ct = tsb_kv_cursor(s->target.kv, q);
        if ((int64_t)fed.size() < ct) return tsb_fail(ctx, TSB_ERR_STATE, "stream %d: the record of fed tokens ends before the cursor", q);
        if (ct + (next_tokens ? 1 : 0) > max_ctx) return tsb_fail(ctx, TSB_ERR_STATE, "stream %d: history beyond the context window", q);
        int32_t* row = s->hist_host.data() + (size_t)a * max_ctx;
        std::copy(fed.begin(), fed.begin() + ct, row);
        int n = (int)ct;
        if (next_tokens) row[n++] = next_tokens[a];
        lens[a] = n;
        lens[n_active + a] = std::min(s->generated[q], n);
    }
    // rows are uploaded at their used length; the copies come from pageable memory, so they are complete when the
    // calls return and hist_host may be reused
    for (int a = 0; a < n_active; a++)
        if (lens[a] > 0)
            TSB_CUDA(ctx, cudaMemcpyAsync(s->hist_dev + (size_t)a * max_ctx, s->hist_host.data() + (size_t)a * max_ctx, (size_t)lens[a] * sizeof(int32_t),
                                          cudaMemcpyHostToDevice, s->stream));
    TSB_CUDA(ctx, cudaMemcpyAsync(s->hist_len_dev, lens, (size_t)n_active * sizeof(int32_t), cudaMemcpyHostToDevice, s->stream));
    TSB_CUDA(ctx, cudaMemcpyAsync(s->gen_dev, lens + n_active, (size_t)n_active * sizeof(int32_t), cudaMemcpyHostToDevice, s->stream));
    return TSB_OK;
}

int32_t session_round_streams(tsb_session* s, const int32_t* streams, int n_active, int k, const tsb_run_config* cfg,
                              int32_t* next_tokens_host, int32_t* accepted_host, int32_t* tokens_out, int32_t* draws_out,
                              uint64_t* draw_step_inout) {
    tsb_ctx* ctx = s->ctx;
    if (!s->has_draft) return tsb_fail(ctx, TSB_ERR_STATE, "the session has no drafter");
    int32_t rc = accept_check_shaping(ctx, &cfg->shaping, true);
    if (rc) return rc;
    const bool penalised = accept_has_penalties(cfg->shaping);
    const int K = k, S = n_active;
    TSB_REQUIRE(ctx, K >= 1 && K <= 15 && K + 1 <= s->max_rows, "block must be 1..15 and fit the session's max_rows");
    TSB_REQUIRE(ctx, S >= 1 && S <= s->n_streams, "bad stream count");
    cudaStream_t st = s->stream;
    const int V = s->target.model->cfg.vocab;
    const double T = cfg->shaping.temperature;
    const bool sampled = T != 0.0;
    for (int a = 0; a < S; a++) {
        const int q = streams[a];
        TSB_REQUIRE(ctx, q >= 0 && q < s->n_streams, "stream %d outside the session", q);
        const int64_t ct = tsb_kv_cursor(s->target.kv, q);
        if (tsb_kv_cursor(s->draft.kv, q) < ct && (rc = drafter_catch_up(s, q, ct))) return rc;  // a lagging drafter replays fed tokens
        const int64_t cd = tsb_kv_cursor(s->draft.kv, q);
        if (ct != cd)
            return tsb_fail(ctx, TSB_ERR_STATE, "stream %d: target cursor %lld and drafter cursor %lld differ", q, (long long)ct,
                            (long long)cd);
    }
    // uniforms: per stream, K draft draws (the row-only step burns one more index), then up to 2K+1 for acceptance
    const int UD = K, UA = 2 * K + 1;
    uint64_t* un = s->uniforms_host;
    for (int a = 0; a < S; a++) {
        const uint64_t seed = cfg->shaping.seed + (uint64_t)streams[a];
        for (int d = 0; d < UD; d++) un[(size_t)a * UD + d] = tsb_uniform_u64(cfg->uniform_mode, seed, draw_step_inout[a] + d);
        for (int j = 0; j < UA; j++)
            un[(size_t)S * UD + (size_t)a * UA + j] = tsb_uniform_u64(cfg->uniform_mode, seed, draw_step_inout[a] + K + 1 + j);
        s->feed_host[(size_t)a * (K + 1)] = next_tokens_host[a];
        // the drafter's first step feeds two rows: the token before the cursor again, then the confirmed one.  After a
        // round in which every proposal was accepted the drafter has never seen the last proposal; feeding the row
        // before the cursor every time keeps the pass shape fixed and replaces the reference's row-only step
        // (crates/runtime/src/speculative.rs:621-623) - a row that is already in the cache is rewritten bit for bit.
        const auto& fed = s->target.fed[streams[a]];
        const int64_t ct = tsb_kv_cursor(s->target.kv, streams[a]);
        if (ct < 1 || (int64_t)fed.size() < ct)
            return tsb_fail(ctx, TSB_ERR_STATE, "stream %d: a round needs at least one fed token before the cursor", streams[a]);
        s->pair_host[2 * a] = fed[(size_t)ct - 1];
        s->pair_host[2 * a + 1] = next_tokens_host[a];
    }
    // a penalised round reads each stream's history - the tokens before the cursor, then the confirmed one - on the device
    if (penalised && (rc = session_stage_history(s, streams, S, next_tokens_host))) return rc;
    const int max_ctx = s->target.model->cfg.max_context;
    uint64_t* un_draft = s->uniforms_dev;
    uint64_t* un_acc = s->uniforms_dev + (size_t)S * UD;
    // pages for every row of the round are reserved up front (a reservation copies the page table synchronously,
    // which must not happen inside a capture), and the shape key of the round is formed
    uint64_t key = 1469598103934665603ull;
    auto mixk = [&](uint64_t v) { key = (key ^ v) * 1099511628211ull; };
    mixk(S), mixk(K), mixk(sampled), mixk(T == 1.0);
    {
        uint64_t tb;
        memcpy(&tb, &T, 8);
        mixk(tb);
        // the truncation settings are kernel parameters of the captured launches
        memcpy(&tb, &cfg->shaping.top_p, 8);
        mixk(tb);
        memcpy(&tb, &cfg->shaping.min_p, 8);
        mixk(tb);
        mixk(cfg->shaping.top_k);
    }
    int64_t max_base = 0;
    for (int a = 0; a < S; a++) {
        const int q = streams[a];
        mixk(q);
        const int64_t base = tsb_kv_cursor(s->target.kv, q);
        if (base + K + 1 > s->target.model->cfg.max_context)
            return tsb_fail(ctx, TSB_ERR_STATE, "stream %d: round of %d rows at %lld exceeds the context window", q, K + 1, (long long)base);
        if ((rc = tsb_kv_reserve(s->target.kv, q, base + K + 1)) || (rc = tsb_kv_reserve(s->draft.kv, q, base + K + 1))) return rc;
        max_base = std::max(max_base, base);
    }
    for (int d = 0; d <= K + 1; d++) mixk((uint64_t)((max_base + d + 1 + 511) / 512));
    s->stage_used = 0;

    auto body = [&]() -> int32_t {
        int32_t rc2;
        if (!s->replay) {
            TSB_CUDA(ctx, cudaMemcpyAsync(s->uniforms_dev, un, (size_t)S * (UD + UA) * sizeof(uint64_t), cudaMemcpyHostToDevice, st));
            TSB_CUDA(ctx, cudaMemcpyAsync(s->feed_dev, s->feed_host, (size_t)S * (K + 1) * sizeof(int32_t), cudaMemcpyHostToDevice, st));
            TSB_CUDA(ctx, cudaMemcpyAsync(s->pair_dev, s->pair_host, (size_t)S * 2 * sizeof(int32_t), cudaMemcpyHostToDevice, st));
            if (!s->capturing) TSB_CUDA(ctx, cudaEventRecord(s->ev[0], st));
        }
        // ---- draft: K steps with a head (crates/runtime/src/speculative.rs:607-659); step 0 carries two rows
        for (int a = 0; a < S; a++) tsb_kv_set_cursor(s->draft.kv, streams[a], tsb_kv_cursor(s->draft.kv, streams[a]) - 1);
        for (int d = 0; d < K; d++) {
            const tsb_row_desc* rd;
            int max_len;
            const int nrow = d == 0 ? 2 : 1;
            if ((rc2 = stage_rows(s, s->draft, streams, S, nrow, nullptr, nullptr, &rd, nullptr, &max_len))) return rc2;
            if (d == 0)
                TSB_CUDA(ctx, forward_device(s, s->draft, s->pair_dev, 1, rd, 2 * S, 2, max_len, s->logits_draft, (int64_t)K * V, true));
            else
                TSB_CUDA(ctx, forward_device(s, s->draft, s->feed_dev + d, K + 1, rd, S, 1, max_len,
                                             s->logits_draft.at((int64_t)d * V), (int64_t)K * V));
            for (int a = 0; a < S; a++) tsb_kv_set_cursor(s->draft.kv, streams[a], tsb_kv_cursor(s->draft.kv, streams[a]) + nrow);
            if (!s->replay) {
                if (penalised)  // every proposal of a round is shaped with the history the round started with (speculative.rs:636-648)
                    TSB_CUDA(ctx, launch_sample_history(ctx, st, s->logits_draft.at((int64_t)d * V), un_draft + d, S, V, cfg->shaping, s->hist_dev, max_ctx,
                                                        s->hist_len_dev, s->gen_dev, s->feed_dev + d + 1, nullptr, s->pen_scratch, (int64_t)K * V, UD,
                                                        K + 1));
                else
                    TSB_CUDA(ctx, launch_sample(ctx, st, s->logits_draft.at((int64_t)d * V), (int64_t)K * V, un_draft + d, UD, S, V, AcceptShape(cfg->shaping),
                                                s->feed_dev + d + 1, K + 1, nullptr, s->accept_scratch));
            }
        }
        if (!s->replay && !s->capturing) TSB_CUDA(ctx, cudaEventRecord(s->ev[1], st));
        // ---- verify: K+1 rows per stream in one pass
        {
            const tsb_row_desc* rd;
            int max_len;
            if ((rc2 = stage_rows(s, s->target, streams, S, K + 1, nullptr, nullptr, &rd, nullptr, &max_len))) return rc2;
            TSB_CUDA(ctx, forward_device(s, s->target, s->feed_dev, 1, rd, S * (K + 1), K + 1, max_len, s->logits_target, V));
        }
        if (!s->replay) {
            if (!s->capturing) TSB_CUDA(ctx, cudaEventRecord(s->ev[2], st));
            // ---- accept on the device; the next confirmed token also lands in feed[.][0]
            if (penalised)
                TSB_CUDA(ctx, launch_accept_history(ctx, st, s->logits_target, s->logits_draft, s->feed_dev + 1, K + 1, un_acc, S, K, V, cfg->shaping,
                                                    s->hist_dev, max_ctx, s->hist_len_dev, s->gen_dev, s->accept_out_dev, s->pen_scratch, s->feed_dev,
                                                    K + 1));
            else
                TSB_CUDA(ctx, launch_accept(ctx, st, s->logits_target, s->logits_draft, s->feed_dev + 1, K + 1, un_acc, S, K, V, AcceptShape(cfg->shaping),
                                            s->accept_out_dev, s->feed_dev, K + 1, s->accept_scratch));
            TSB_CUDA(ctx, cudaMemcpyAsync(s->accept_out_host, s->accept_out_dev, (size_t)S * sizeof(tsb_accept_out),
                                          cudaMemcpyDeviceToHost, st));
            if (!s->capturing) TSB_CUDA(ctx, cudaEventRecord(s->ev[3], st));
        }
        return TSB_OK;
    };

    // A round that fails part-way (a refused staging, a failed capture) must not leave the two caches out of step:
    // the cursors the body moves are put back on any error, so the caller can call again or discard.
    std::vector<int64_t> cur_t(S), cur_d(S);
    for (int a = 0; a < S; a++) cur_t[a] = tsb_kv_cursor(s->target.kv, streams[a]), cur_d[a] = tsb_kv_cursor(s->draft.kv, streams[a]);
    auto restore = [&](int32_t code) {
        for (int a = 0; a < S; a++) tsb_kv_set_cursor(s->target.kv, streams[a], cur_t[a]), tsb_kv_set_cursor(s->draft.kv, streams[a], cur_d[a]);
        s->stage_used = 0;
        return code;
    };
    const bool want_graph = s->use_graph && s->rounds_done >= 1 && !penalised;
    if (want_graph && s->graph && s->graph_key == key) {
        s->replay = true;  // host-side staging only: descriptors land in the pinned ring at the captured offsets
        rc = body();
        s->replay = false;
        if (rc) return restore(rc);
        TSB_CUDA(ctx, cudaEventRecord(s->ev[0], st));
        TSB_CUDA(ctx, cudaGraphLaunch(s->graph, st));
        TSB_CUDA(ctx, cudaEventRecord(s->ev[3], st));
        ctx->launches += s->graph_launches;
        s->last_round_graphed = true;
    } else if (want_graph) {
        if (s->graph) cudaGraphExecDestroy(s->graph), s->graph = nullptr;
        const uint64_t l0 = ctx->launches;
        TSB_CUDA(ctx, cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal));
        s->capturing = true;
        rc = body();
        s->capturing = false;
        cudaGraph_t g = nullptr;
        cudaError_t ce = cudaStreamEndCapture(st, &g);
        if (rc) {
            if (g) cudaGraphDestroy(g);
            return restore(rc);
        }
        if (ce != cudaSuccess) return restore(tsb_fail(ctx, TSB_ERR_CUDA, "ending the capture of a round failed: %s", cudaGetErrorString(ce)));
        ce = cudaGraphInstantiate(&s->graph, g, 0);
        cudaGraphDestroy(g);
        if (ce != cudaSuccess) {
            s->graph = nullptr;
            return restore(tsb_fail(ctx, TSB_ERR_CUDA, "instantiating the graph of a round failed: %s", cudaGetErrorString(ce)));
        }
        s->graph_key = key;
        s->graph_launches = ctx->launches - l0;
        TSB_CUDA(ctx, cudaEventRecord(s->ev[0], st));
        TSB_CUDA(ctx, cudaGraphLaunch(s->graph, st));
        TSB_CUDA(ctx, cudaEventRecord(s->ev[3], st));
        s->last_round_graphed = true;
    } else {
        if ((rc = body())) {
            cudaStreamSynchronize(st);  // what was enqueued before the failure is over before the cursors move back
            return restore(rc);
        }
        s->last_round_graphed = false;
    }
    s->rounds_done++;
    if ((rc = tsb_stream_sync(ctx, st))) return restore(rc);
    s->stage_used = 0;
    // ---- commit: cursors to the accepted prefix (rollback_retaining + rewind_drafter)
    for (int a = 0; a < S; a++) {
        const int q = streams[a];
        const tsb_accept_out& o = s->accept_out_host[a];
        if (o.status != 0)
            return tsb_fail(ctx, TSB_ERR_DEVICE, "stream %d: a logit was not finite or a proposal was out of range", q);
        const int64_t base = tsb_kv_cursor(s->target.kv, q);
        auto& fed = s->target.fed[q];
        fed.resize((size_t)base);
        fed.push_back(next_tokens_host[a]);
        for (int i = 0; i < o.accepted; i++) fed.push_back(o.tokens[i]);
        tsb_kv_set_cursor(s->target.kv, q, base + o.accepted + 1);
        tsb_kv_set_cursor(s->draft.kv, q, base + o.accepted + 1);
        accepted_host[a] = o.accepted;
        if (tokens_out) memcpy(tokens_out + (size_t)a * 16, o.tokens, sizeof(o.tokens));
        if (draws_out) draws_out[a] = o.draws;
        next_tokens_host[a] = o.tokens[o.accepted];
        s->generated[q] += o.accepted + 1;  // the accepted proposals and the token that enters the next round
        draw_step_inout[a] += (sampled ? (uint64_t)(K + 1) : 0) + (uint64_t)o.draws;
    }
    return TSB_OK;
}

int32_t session_stage_ints(tsb_session* s, const int32_t* data, int n, const int32_t** dev) {
    tsb_ctx* ctx = s->ctx;
    TSB_REQUIRE(ctx, n <= s->stage_int_cap, "%d integers exceed the staging ring's %d", n, s->stage_int_cap);
    if (s->stage_int_used + n > s->stage_int_cap) {
        TSB_CUDA(ctx, cudaStreamSynchronize(s->stream));
        s->stage_int_used = 0;
    }
    std::copy(data, data + n, s->stage_int_host + s->stage_int_used);
    *dev = s->stage_int_dev + s->stage_int_used;
    if (n > 0)
        TSB_CUDA(ctx, cudaMemcpyAsync(s->stage_int_dev + s->stage_int_used, s->stage_int_host + s->stage_int_used, (size_t)n * sizeof(int32_t),
                                      cudaMemcpyHostToDevice, s->stream));
    s->stage_int_used += (n + 3) / 4 * 4;
    return TSB_OK;
}

int32_t session_ragged_pass(tsb_session* s, const RowGroup* groups, int n_groups, const int32_t* tokens, int rows, const int32_t* want_rows, int n_want) {
    tsb_ctx* ctx = s->ctx;
    ModelRt& rt = s->target;
    TSB_REQUIRE(ctx, rt.model->family->ragged, "%s models take no mixed passes", rt.model->family->name);
    TSB_REQUIRE(ctx, rows > 0 && rows <= s->pass_rows && n_want <= s->logit_rows, "a pass of %d rows with %d logit rows exceeds the session's %d and %d",
                rows, n_want, s->pass_rows, s->logit_rows);
    Pass p;
    for (int i = 0; i < n_groups; i++) {
        const RowGroup& g = groups[i];
        TSB_REQUIRE(ctx, g.seq >= 0 && g.seq < s->n_streams && g.n_rows > 0 && g.first_row >= 0 && g.first_row + g.n_rows <= rows, "bad group %d", i);
        if (g.base != tsb_kv_cursor(rt.kv, g.seq)) return tsb_fail(ctx, TSB_ERR_STATE, "stream %d does not continue at %lld", g.seq, (long long)g.base);
        if (g.base + g.n_rows > rt.model->cfg.max_context)
            return tsb_fail(ctx, TSB_ERR_STATE, "stream %d: %lld + %d rows exceed the context window %d", g.seq, (long long)g.base, g.n_rows,
                            rt.model->cfg.max_context);
        int32_t rc = tsb_kv_reserve(rt.kv, g.seq, g.base + g.n_rows);
        if (rc) return rc;
        p.max_len = std::max(p.max_len, (int)g.base + g.n_rows);
    }
    if (s->stage_used + rows > s->stage_cap) {
        TSB_CUDA(ctx, cudaStreamSynchronize(s->stream));
        s->stage_used = 0;
    }
    tsb_row_desc* hd = s->stage_rows_host + s->stage_used;
    int32_t* ht = s->stage_tok_host + s->stage_used;
    for (int i = 0; i < n_groups; i++)
        for (int j = 0; j < groups[i].n_rows; j++) {
            tsb_row_desc& d = hd[groups[i].first_row + j];
            d.seq = groups[i].seq, d.base = (int32_t)groups[i].base, d.slot = j, d.position = (int32_t)groups[i].base + j;
            d.mask[0] = d.mask[1] = 0;  // chains: a row sees every earlier position
        }
    std::copy(tokens, tokens + rows, ht);
    p.rows_dev = s->stage_rows_dev + s->stage_used, p.tokens = s->stage_tok_dev + s->stage_used;
    TSB_CUDA(ctx, cudaMemcpyAsync(s->stage_rows_dev + s->stage_used, hd, rows * sizeof(tsb_row_desc), cudaMemcpyHostToDevice, s->stream));
    TSB_CUDA(ctx, cudaMemcpyAsync(s->stage_tok_dev + s->stage_used, ht, rows * sizeof(int32_t), cudaMemcpyHostToDevice, s->stream));
    s->stage_used += rows;
    if (n_want > 0) {
        int32_t rc = session_stage_ints(s, want_rows, n_want, &p.want_dev);
        if (rc) return rc;
        p.logits = s->logits_target, p.logits_stride = rt.model->cfg.vocab, p.n_want = n_want;
    }
    p.rows = rows, p.groups = groups, p.n_groups = n_groups;
    TSB_CUDA(ctx, rt.model->family->forward(s, rt, p));
    for (int i = 0; i < n_groups; i++) {
        record_fed(rt, groups[i].seq, groups[i].base, tokens + groups[i].first_row, groups[i].n_rows);
        tsb_kv_set_cursor(rt.kv, groups[i].seq, groups[i].base + groups[i].n_rows);
    }
    return TSB_OK;
}

int32_t session_prefill_rows(tsb_session* s, int stream, const int32_t* tokens, int n) {
    TSB_REQUIRE(s->ctx, stream >= 0 && stream < s->n_streams, "stream %d outside the session", stream);
    if (s->target.model->family->ragged) {  // portions as large as a pass may be
        for (int i = 0; i < n; i += s->pass_rows) {
            const RowGroup g{stream, 0, std::min(s->pass_rows, n - i), tsb_kv_cursor(s->target.kv, stream)};
            int32_t rc = session_ragged_pass(s, &g, 1, tokens + i, g.n_rows, nullptr, 0);
            if (rc) return rc;
        }
        return TSB_OK;
    }
    const int chunk = std::min(s->max_rows, 64);
    for (int i = 0; i < n; i += chunk) {
        const int m = std::min(chunk, n - i);
        const int64_t pos = tsb_kv_cursor(s->target.kv, stream);
        record_fed(s->target, stream, pos, tokens + i, m);
        int32_t rc = forward_stream(s, s->target, stream, tokens + i, m, nullptr, LogitRows(), nullptr);
        if (rc) return rc;
    }
    return TSB_OK;
}

// ---- tree drafting (crates/runtime/src/speculative.rs:461-560; tree shape helpers runtime/src/dflash_tree.rs)
// The drafter runs over every slot drafted so far (tree mask) and its logits at the rows that get children give
// those children: simple rather than fast - a level (static shape) or an expansion (best-first) costs one pass.
static int32_t drafter_children(tsb_session* s, int stream, const std::vector<int32_t>& feed, const std::vector<int32_t>& slot_parent, int n_known,
                                const std::vector<int32_t>& rows, int width, bool want_scores, std::vector<int32_t>& child,
                                std::vector<float>& scores) {
    tsb_ctx* ctx = s->ctx;
    const int V = s->target.model->cfg.vocab;
    const int64_t base = tsb_kv_cursor(s->draft.kv, stream);
    int32_t rc = forward_stream(s, s->draft, stream, feed.data(), n_known, slot_parent.data(), s->logits_draft, nullptr);
    if (rc) return rc;
    tsb_kv_set_cursor(s->draft.kv, stream, base);
    int32_t* rows_dev = s->tree_dev;  // row list (128 ints), then eight picks per row
    int32_t* child_dev = s->tree_dev + 128;
    const int nr = (int)rows.size();
    child.assign((size_t)nr * 8, -1);
    TSB_CUDA(ctx, cudaMemcpyAsync(rows_dev, rows.data(), nr * sizeof(int32_t), cudaMemcpyHostToDevice, s->stream));
    TSB_CUDA(ctx, launch_topk_rows(ctx, s->stream, (const __half*)s->logits_draft.p, V, rows_dev, nr, width, child_dev));
    TSB_CUDA(ctx, cudaMemcpyAsync(child.data(), child_dev, (size_t)nr * 8 * sizeof(int32_t), cudaMemcpyDeviceToHost, s->stream));
    if ((rc = tsb_stream_sync(ctx, s->stream))) return rc;
    for (int r = 0; r < nr; r++)
        for (int c = 0; c < width; c++)
            if (child[(size_t)r * 8 + c] < 0) return tsb_fail(ctx, TSB_ERR_DEVICE, "the drafter's logits at tree slot %d are not finite", rows[r]);
    if (want_scores) {
        // the picked candidates' logits, the scores the best-first builder's softmax runs over
        std::vector<uint16_t> raw((size_t)nr * width);
        for (int r = 0; r < nr; r++)
            for (int c = 0; c < width; c++)
                TSB_CUDA(ctx, cudaMemcpyAsync(&raw[(size_t)r * width + c], (const __half*)s->logits_draft.p + (size_t)rows[r] * V + child[(size_t)r * 8 + c], 2,
                                              cudaMemcpyDeviceToHost, s->stream));
        if ((rc = tsb_stream_sync(ctx, s->stream))) return rc;
        scores.resize(raw.size());
        for (size_t i = 0; i < raw.size(); i++) scores[i] = __half2float(__ushort_as_half(raw[i]));
    }
    return TSB_OK;
}

int32_t session_draft_tree(tsb_session* s, int stream, const TreeShape& shape, int32_t next, int64_t base, std::vector<int32_t>& feed,
                           std::vector<int32_t>& slot_parent, std::vector<tsb_tree_node>& nodes, int* drafter_rows) {
    tsb_ctx* ctx = s->ctx;
    if (!s->has_draft) return tsb_fail(ctx, TSB_ERR_STATE, "the session has no drafter");
    const int N = shape.nodes, LV = shape.levels;
    TSB_REQUIRE(ctx, N >= 1 && N + 1 <= s->max_rows && N + 1 <= 128, "tree of %d nodes + anchor exceeds the session's %d rows", N, s->max_rows);
    TSB_REQUIRE(ctx, LV >= 1 && LV <= 8, "tree_levels must be 1..8");
    int32_t rc;
    if (tsb_kv_cursor(s->draft.kv, stream) < base && (rc = drafter_catch_up(s, stream, base))) return rc;
    if (tsb_kv_cursor(s->draft.kv, stream) != base)
        return tsb_fail(ctx, TSB_ERR_STATE, "tree draft at %lld: drafter cursor %lld", (long long)base, (long long)tsb_kv_cursor(s->draft.kv, stream));
    if (base + N + 1 > s->draft.model->cfg.max_context) return tsb_fail(ctx, TSB_ERR_STATE, "a tree of %d rows at %lld exceeds the context window", N + 1, (long long)base);
    nodes.clear();
    feed.assign(1, next);
    slot_parent.assign(1, -1);
    std::vector<int32_t> child;
    std::vector<float> sc;
    int drafted = 0;
    if (shape.best_first) {
        TSB_REQUIRE(ctx, shape.cand >= 1 && shape.cand <= 8, "tree_cand must be 1..8");
        // children of node `parent` (the anchor for -1): the drafter's `cand` most likely tokens after it, scored by
        // their logits.  The expanded node is always the newest slot, so one pass over the slots so far gives its row.
        std::vector<std::vector<int32_t>> cand_tokens;  // per expanded parent (index parent + 1): its candidates' tokens
        cand_tokens.resize((size_t)N + 1);
        std::vector<tsb_tree_node> out;
        // best_first_tree appends a node and, when it has room, expands it at once: `out` is mirrored in feed/slot_parent
        // inside the callback, which therefore sees every earlier node's slot already in place
        std::vector<tsb_tree_node> seen;
        // The builder is run step by step here (instead of through the callback form) because a node's token is only
        // known once its parent's candidates have been scored.
        struct Front {
            double p;
            tsb_tree_node n;
        };
        std::vector<Front> frontier;
        auto expand = [&](int depth, int parent, double path_p) -> int32_t {
            const int n_known = (int)feed.size();
            std::vector<int32_t> rows{parent + 1};
            int32_t rc2 = drafter_children(s, stream, feed, slot_parent, n_known, rows, shape.cand, true, child, sc);
            if (rc2) return rc2;
            drafted = n_known;
            cand_tokens[(size_t)parent + 1].assign(child.begin(), child.begin() + shape.cand);
            float mf = -INFINITY;
            for (int i = 0; i < shape.cand; i++) mf = fmaxf(mf, sc[i]);
            const double m = (double)mf;
            double e[8], z = 0.0;
            for (int i = 0; i < shape.cand; i++) e[i] = exp((double)sc[i] - m);
            for (int i = 0; i < shape.cand; i++) z += e[i];
            for (int c = 0; c < shape.cand; c++) frontier.push_back({path_p * (e[c] / z), tsb_tree_node{depth, c, parent}});
            return TSB_OK;
        };
        if ((rc = expand(0, -1, 1.0))) return rc;
        while ((int)nodes.size() < N && !frontier.empty()) {
            size_t best = 0;
            for (size_t i = 1; i < frontier.size(); i++) {
                const Front &f = frontier[i], &b = frontier[best];
                if (f.p > b.p || (f.p == b.p && (f.n.depth < b.n.depth || (f.n.depth == b.n.depth && f.n.cand < b.n.cand)))) best = i;
            }
            const Front picked = frontier[best];
            frontier[best] = frontier.back();
            frontier.pop_back();
            const int id = (int)nodes.size();
            nodes.push_back(picked.n);
            feed.push_back(cand_tokens[(size_t)picked.n.parent + 1][picked.n.cand]);
            slot_parent.push_back(picked.n.parent + 1);
            if ((int)nodes.size() < N && picked.n.depth + 1 < LV && (rc = expand(picked.n.depth + 1, id, picked.p))) return rc;
        }
        *drafter_rows = drafted;
        return TSB_OK;
    }
    for (int l = 0; l < LV; l++) TSB_REQUIRE(ctx, shape.branching[l] >= 1 && shape.branching[l] <= 8, "tree_branching must be 1..8");
    // the static shape, breadth-first, cut at N nodes: slot 0 is the anchor, node i sits in slot i + 1
    std::vector<int> level_begin{0, 1};  // slots of level l are [level_begin[l], level_begin[l+1])
    std::vector<int> depth_of{0}, cand_of{0};
    for (int l = 0; l < LV && (int)slot_parent.size() < N + 1; l++) {
        const int lo = level_begin[l], hi = level_begin[l + 1];
        for (int p = lo; p < hi && (int)slot_parent.size() < N + 1; p++)
            for (int c = 0; c < shape.branching[l] && (int)slot_parent.size() < N + 1; c++) {
                slot_parent.push_back(p);
                depth_of.push_back(l), cand_of.push_back(c);
            }
        level_begin.push_back((int)slot_parent.size());
    }
    const int rows = (int)slot_parent.size();
    TSB_REQUIRE(ctx, rows == N + 1, "the branching list yields %d nodes, fewer than tree_nodes %d", rows - 1, N);
    feed.resize(rows, 0);
    for (int i = 1; i < rows; i++) nodes.push_back(tsb_tree_node{depth_of[i], cand_of[i], slot_parent[i] - 1});
    const int n_levels = (int)level_begin.size() - 1;  // levels that hold slots (anchor level included)
    std::vector<int32_t> row_ids;
    for (int l = 0; l + 1 < n_levels; l++) {
        const int n = level_begin[l + 1];  // slots 0 .. n-1 are known
        const int lo = level_begin[l], hi = level_begin[l + 1];
        row_ids.resize(hi - lo);
        for (int p = lo; p < hi; p++) row_ids[p - lo] = p;
        if ((rc = drafter_children(s, stream, feed, slot_parent, n, row_ids, shape.branching[l], false, child, sc))) return rc;
        drafted = n;
        int slot = level_begin[l + 1];  // children of the level's nodes, in slot order
        for (int p = lo; p < hi; p++)
            for (int c = 0; c < shape.branching[l] && slot < level_begin[l + 2]; c++, slot++) feed[slot] = child[(size_t)(p - lo) * 8 + c];
    }
    *drafter_rows = drafted;
    return TSB_OK;
}

// ---- tree round: draft, then anchor + nodes in one target pass and the target's pick at every row
int32_t session_tree_round(tsb_session* s, int stream, const tsb_run_config* cfg, int32_t next, int64_t base,
                           std::vector<int32_t>& feed, std::vector<int32_t>& slot_parent, std::vector<int32_t>& picks,
                           int* drafter_rows) {
    tsb_ctx* ctx = s->ctx;
    TSB_REQUIRE(ctx, cfg->shaping.temperature == 0.0, "tree rounds need temperature 0 (sampled tree acceptance is not defined)");
    TreeShape shape;
    shape.nodes = cfg->tree_nodes, shape.levels = cfg->tree_levels, shape.best_first = cfg->tree_best_first, shape.cand = cfg->tree_cand;
    for (int l = 0; l < 8; l++) shape.branching[l] = cfg->tree_branching[l];
    const int V = s->target.model->cfg.vocab;
    if (tsb_kv_cursor(s->target.kv, stream) != base)
        return tsb_fail(ctx, TSB_ERR_STATE, "tree round at %lld: target cursor %lld", (long long)base, (long long)tsb_kv_cursor(s->target.kv, stream));
    std::vector<tsb_tree_node> nodes;
    int32_t rc = session_draft_tree(s, stream, shape, next, base, feed, slot_parent, nodes, drafter_rows);
    if (rc) return rc;
    const int rows = (int)feed.size();
    if ((rc = forward_stream(s, s->target, stream, feed.data(), rows, slot_parent.data(), s->logits_target, nullptr))) return rc;
    tsb_kv_set_cursor(s->target.kv, stream, base);
    TSB_REQUIRE(ctx, (size_t)rows * accept_row_stats_bytes() <= s->accept_scratch_bytes, "tree of %d rows exceeds the acceptance scratch", rows);
    TSB_CUDA(ctx, launch_argmax_rows(ctx, s->stream, s->logits_target, rows, V, s->accept_scratch));
    std::vector<uint8_t> stats((size_t)rows * accept_row_stats_bytes());
    TSB_CUDA(ctx, cudaMemcpyAsync(stats.data(), s->accept_scratch, stats.size(), cudaMemcpyDeviceToHost, s->stream));
    if ((rc = tsb_stream_sync(ctx, s->stream))) return rc;
    picks.resize(rows);
    for (int r = 0; r < rows; r++) {
        int32_t am, bad;
        accept_row_stats_read(stats.data(), r, &am, &bad);
        if (bad) return tsb_fail(ctx, TSB_ERR_DEVICE, "a target logit at tree slot %d is not finite", r);
        picks[r] = am;
    }
    return TSB_OK;
}

int32_t session_tree_commit(tsb_session* s, int stream, int64_t base, const std::vector<int32_t>& feed,
                            const std::vector<uint32_t>& path, int keep, int drafter_rows) {
    tsb_ctx* ctx = s->ctx;
    int32_t rc = tsb_kv_commit_path(ctx, s->stream, s->target.kv, stream, base, path.data(), keep);
    if (rc) return rc;
    // the drafter holds rows only for the slots it was run over: keep the part of the path it has, the rest is
    // replayed from the record of fed tokens before its next step
    int dkeep = 0;
    while (dkeep < keep && (int)path[dkeep] < drafter_rows) dkeep++;
    if (dkeep > 0 && (rc = tsb_kv_commit_path(ctx, s->stream, s->draft.kv, stream, base, path.data(), dkeep))) return rc;
    if ((rc = tsb_stream_sync(ctx, s->stream))) return rc;
    tsb_kv_set_cursor(s->target.kv, stream, base + keep);
    tsb_kv_set_cursor(s->draft.kv, stream, base + dkeep);
    auto& fed = s->target.fed[stream];
    fed.resize((size_t)base);
    for (int r = 0; r < keep; r++) fed.push_back(feed[path[r]]);
    return TSB_OK;
}

int32_t session_select_target(tsb_session* s, int stream, const tsb_run_config* cfg, uint64_t uniform, int32_t* token_host) {
    tsb_ctx* ctx = s->ctx;
    const int V = s->target.model->cfg.vocab;
    int32_t rc = accept_check_shaping(ctx, &cfg->shaping, true);
    if (rc) return rc;
    uint64_t* u = s->uniforms_host;
    u[0] = uniform;
    TSB_CUDA(ctx, cudaMemcpyAsync(s->uniforms_dev, u, sizeof(uint64_t), cudaMemcpyHostToDevice, s->stream));
    if (accept_has_penalties(cfg->shaping)) {
        // select(logits, shaping, history): the history is everything fed so far (crates/selection/src/choose.rs:139-154)
        if ((rc = session_stage_history(s, &stream, 1, nullptr))) return rc;
        TSB_CUDA(ctx, launch_sample_history(ctx, s->stream, s->logits_target, s->uniforms_dev, 1, V, cfg->shaping, s->hist_dev,
                                            s->target.model->cfg.max_context, s->hist_len_dev, s->gen_dev, s->tok1_dev, nullptr, s->pen_scratch));
    } else {
        TSB_CUDA(ctx, launch_sample(ctx, s->stream, s->logits_target, V, s->uniforms_dev, 1, 1, V, AcceptShape(cfg->shaping),
                                    s->tok1_dev, 1, nullptr, s->accept_scratch));
    }
    TSB_CUDA(ctx, cudaMemcpyAsync(s->feed_host, s->tok1_dev, sizeof(int32_t), cudaMemcpyDeviceToHost, s->stream));
    if ((rc = tsb_stream_sync(ctx, s->stream))) return rc;
    *token_host = s->feed_host[0];
    return TSB_OK;
}

extern "C" {

int32_t tsb_session_round(tsb_session* s, const tsb_run_config* cfg, int32_t* next_tokens_host, int32_t* accepted_host,
                          uint64_t* draw_step_inout) {
    if (!s || !cfg || !next_tokens_host || !accepted_host || !draw_step_inout) return TSB_ERR_INVALID;
    DeviceGuard g(s->ctx);
    std::vector<int32_t> streams(s->n_streams);
    for (int q = 0; q < s->n_streams; q++) streams[q] = q;
    return session_round_streams(s, streams.data(), s->n_streams, cfg->block, cfg, next_tokens_host, accepted_host, nullptr,
                                 nullptr, draw_step_inout);
}

int32_t tsb_session_round_tokens(tsb_session* s, const tsb_run_config* cfg, int32_t* next_tokens_host, int32_t* accepted_host,
                                 int32_t* tokens_out, uint64_t* draw_step_inout) {
    if (!s || !cfg || !next_tokens_host || !accepted_host || !tokens_out || !draw_step_inout) return TSB_ERR_INVALID;
    DeviceGuard g(s->ctx);
    std::vector<int32_t> streams(s->n_streams);
    for (int q = 0; q < s->n_streams; q++) streams[q] = q;
    return session_round_streams(s, streams.data(), s->n_streams, cfg->block, cfg, next_tokens_host, accepted_host, tokens_out,
                                 nullptr, draw_step_inout);
}

int32_t tsb_session_step(tsb_session* s, const tsb_step_entry* entries, int32_t n_entries, const int32_t* tokens, const int32_t* want,
                         void* logits_out_host) {
    if (!s || !entries || !tokens) return TSB_ERR_INVALID;
    tsb_ctx* ctx = s->ctx;
    ModelRt& rt = s->target;
    TSB_REQUIRE(ctx, n_entries > 0, "a step has entries");
    DeviceGuard g(ctx);
    const int V = rt.model->cfg.vocab;
    std::vector<char> seen(s->n_streams, 0);
    int64_t total_want = 0, need = 0;
    for (int i = 0, wi = 0; i < n_entries; i++) {
        const tsb_step_entry& e = entries[i];
        TSB_REQUIRE(ctx, e.stream >= 0 && e.stream < s->n_streams && !seen[e.stream], "entry %d: stream %d is outside the session or comes twice", i, e.stream);
        TSB_REQUIRE(ctx, e.n_tokens > 0 && e.n_want >= 0 && e.n_want <= e.n_tokens, "entry %d: bad token or want count", i);
        seen[e.stream] = 1;
        for (int k = 0; k < e.n_want; k++, wi++)
            TSB_REQUIRE(ctx, want && want[wi] >= 0 && want[wi] < e.n_tokens && (k == 0 || want[wi] > want[wi - 1]), "entry %d: wanted places ascend inside its tokens", i);
        total_want += e.n_want;
        const int64_t end = tsb_kv_cursor(rt.kv, e.stream) + e.n_tokens;
        if (end > rt.model->cfg.max_context)
            return tsb_fail(ctx, TSB_ERR_STATE, "stream %d: %lld positions exceed the context window %d", e.stream, (long long)end, rt.model->cfg.max_context);
        const KvView& v = rt.kv->view;
        need += std::max<int64_t>(0, ((end + v.page_tokens - 1) >> v.page_shift) - rt.kv->pages_of_seq[e.stream]);
    }
    TSB_REQUIRE(ctx, total_want == 0 || logits_out_host, "wanted logits need a buffer");
    if (need > (int64_t)rt.kv->free_pages.size())
        return tsb_fail(ctx, TSB_ERR_OOM, "the step needs %lld pages, %zu are free", (long long)need, rt.kv->free_pages.size());
    char* out = static_cast<char*>(logits_out_host);
    const size_t row_bytes = (size_t)V * s->logits_target.bytes();
    if (!rt.model->family->ragged) {
        // stream by stream, in portions of the largest uniform pass
        for (int i = 0; i < n_entries; tokens += entries[i].n_tokens, i++) {
            const tsb_step_entry& e = entries[i];
            int wi = 0;
            for (int t = 0; t < e.n_tokens; t += s->max_rows) {
                const int n = std::min(s->max_rows, e.n_tokens - t);
                record_fed(rt, e.stream, tsb_kv_cursor(rt.kv, e.stream), tokens + t, n);
                const bool head = wi < e.n_want && want[wi] < t + n;
                int32_t rc = forward_stream(s, rt, e.stream, tokens + t, n, nullptr, head ? s->logits_target : LogitRows(), nullptr);
                if (rc) return rc;
                for (; wi < e.n_want && want[wi] < t + n; wi++, out += row_bytes)
                    TSB_CUDA(ctx, cudaMemcpyAsync(out, s->logits_target.at((int64_t)(want[wi] - t) * V).p, row_bytes, cudaMemcpyDeviceToHost, s->stream));
            }
            want += e.n_want;
        }
        return tsb_stream_sync(ctx, s->stream);
    }
    // one batch; cut only where it exceeds what a pass holds
    std::vector<RowGroup> groups;
    std::vector<int32_t> feed, rows_wanted;
    auto flush = [&]() -> int32_t {
        if (feed.empty()) return TSB_OK;
        int32_t rc = session_ragged_pass(s, groups.data(), (int)groups.size(), feed.data(), (int)feed.size(), rows_wanted.data(), (int)rows_wanted.size());
        if (rc) return rc;
        if (!rows_wanted.empty()) {
            TSB_CUDA(ctx, cudaMemcpyAsync(out, s->logits_target.p, rows_wanted.size() * row_bytes, cudaMemcpyDeviceToHost, s->stream));
            if ((rc = tsb_stream_sync(ctx, s->stream))) return rc;
            out += rows_wanted.size() * row_bytes;
        }
        groups.clear(), feed.clear(), rows_wanted.clear();
        return TSB_OK;
    };
    int32_t rc;
    for (int i = 0, wi = 0; i < n_entries; tokens += entries[i].n_tokens, i++) {
        const tsb_step_entry& e = entries[i];
        const int w_end = wi + e.n_want;
        bool open = false;
        for (int t = 0; t < e.n_tokens; t++) {
            const bool w = wi < w_end && want[wi] == t;
            if ((int)feed.size() == s->pass_rows || (w && (int)rows_wanted.size() == s->logit_rows)) {
                if ((rc = flush())) return rc;
                open = false;
            }
            if (!open) groups.push_back({e.stream, (int)feed.size(), 0, tsb_kv_cursor(rt.kv, e.stream)}), open = true;
            groups.back().n_rows++;
            if (w) rows_wanted.push_back((int32_t)feed.size()), wi++;
            feed.push_back(tokens[t]);
        }
    }
    if ((rc = flush())) return rc;
    return tsb_stream_sync(ctx, s->stream);
}

void* tsb_session_stream(tsb_session* s) { return s ? (void*)s->stream : nullptr; }

int32_t tsb_session_set_graph(tsb_session* s, int32_t enabled) {
    if (!s) return TSB_ERR_INVALID;
    s->use_graph = enabled != 0;
    return TSB_OK;
}

int32_t tsb_session_round_times(tsb_session* s, float* out4_ms) {
    if (!s || !out4_ms) return TSB_ERR_INVALID;
    DeviceGuard g(s->ctx);
    // a graphed round has no event records inside it: only the total (index 3) is known
    for (int i = 0; i < 3; i++) {
        out4_ms[i] = -1.f;
        if (!s->last_round_graphed && cudaEventElapsedTime(&out4_ms[i], s->ev[i], s->ev[i + 1]) != cudaSuccess) out4_ms[i] = -1.f;
    }
    if (cudaEventElapsedTime(&out4_ms[3], s->ev[0], s->ev[3]) != cudaSuccess) out4_ms[3] = -1.f;
    cudaGetLastError();
    return TSB_OK;
}

}  // extern "C"
