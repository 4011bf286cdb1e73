// Continuous batching over a session's streams: requests of unequal prompts and budgets share every step.
//
// A request owns a stream and the pages for its prompt and budget from admission to its end, so a step never runs out of
// pages.  A step carries one token of every decoding request and, in the rows that are left, prompt portions in admission
// order; the last row of every request that ends its prompt or decodes gets logits, and all of those are sampled on the
// device by one launch.  Draw indices, stop tokens and budgets follow the sequential loop of spec_loop.cu.
#include <algorithm>
#include <chrono>
#include <deque>
#include <vector>

#include "accept.cuh"
#include "model.cuh"

namespace {

struct Live {
    int request = -1, stream = -1;
    const int32_t* prompt = nullptr;
    int n_prompt = 0, fed = 0;  // prompt tokens fed so far
    int budget = 0, generated = 0;
    int32_t next = -1;          // the sampled token that the next step feeds
};

double now_s() { return std::chrono::duration<double>(std::chrono::steady_clock::now().time_since_epoch()).count(); }

// tokens[i] = draw from logit row i with the history of live[i]'s stream
int32_t sample_rows(tsb_session* s, const std::vector<const Live*>& who, const tsb_run_config* cfg, std::vector<int32_t>& tokens) {
    tsb_ctx* ctx = s->ctx;
    const int n = (int)who.size(), V = s->target.model->cfg.vocab;
    std::vector<int32_t> streams(n);
    for (int i = 0; i < n; i++) {
        const Live& l = *who[i];
        streams[i] = l.stream;
        const uint64_t seed = cfg->shaping.seed + (uint64_t)l.request;
        const uint64_t step = cfg->uniform_mode == 0 ? (uint64_t)l.generated : (1ull << 63) + (uint64_t)l.generated;
        s->uniforms_host[i] = tsb_uniform_u64(cfg->uniform_mode, seed, step);
        s->generated[l.stream] = l.generated;
    }
    TSB_CUDA(ctx, cudaMemcpyAsync(s->uniforms_dev, s->uniforms_host, n * sizeof(uint64_t), cudaMemcpyHostToDevice, s->stream));
    if (accept_has_penalties(cfg->shaping)) {
        int32_t rc = session_stage_history(s, streams.data(), n, nullptr);
        if (rc) return rc;
        TSB_CUDA(ctx, launch_sample_history(ctx, s->stream, s->logits_target, s->uniforms_dev, n, V, cfg->shaping, s->hist_dev,
                                            s->target.model->cfg.max_context, s->hist_len_dev, s->gen_dev, s->tok1_dev, nullptr, s->pen_scratch));
    } else {
        TSB_CUDA(ctx, launch_sample(ctx, s->stream, s->logits_target, V, s->uniforms_dev, 1, n, V, AcceptShape(cfg->shaping), s->tok1_dev, 1, nullptr,
                                    s->accept_scratch));
    }
    tokens.resize(n);
    TSB_CUDA(ctx, cudaMemcpyAsync(s->feed_host, s->tok1_dev, n * sizeof(int32_t), cudaMemcpyDeviceToHost, s->stream));
    int32_t rc = tsb_stream_sync(ctx, s->stream);
    if (rc) return rc;
    std::copy(s->feed_host, s->feed_host + n, tokens.begin());
    return TSB_OK;
}

}  // namespace

extern "C" int32_t tsb_serve_run(tsb_session* s, const tsb_serve_request* requests, int32_t n_requests, const int32_t* prompts, const tsb_run_config* cfg,
                                 int32_t prefill_chunk, int32_t* out_tokens, int32_t out_stride, int32_t* out_counts, int32_t* out_reasons,
                                 tsb_serve_stats* stats) {
    if (!s || !requests || !prompts || !cfg || !out_tokens || !out_counts || !out_reasons) return TSB_ERR_INVALID;
    tsb_ctx* ctx = s->ctx;
    ModelRt& rt = s->target;
    if (!rt.model->family->ragged) return tsb_fail(ctx, TSB_ERR_UNSUPPORTED, "%s models take no mixed passes", rt.model->family->name);
    int32_t rc = accept_check_shaping(ctx, &cfg->shaping, true);
    if (rc) return rc;
    TSB_REQUIRE(ctx, n_requests > 0 && prefill_chunk > 0, "requests and a positive portion size expected");
    TSB_REQUIRE(ctx, s->pass_rows > s->n_streams || prefill_chunk == 1, "a pass of %d rows leaves no room for prompts beside %d decoding streams", s->pass_rows, s->n_streams);
    DeviceGuard g(ctx);
    const KvView& v = rt.kv->view;
    const int max_ctx = rt.model->cfg.max_context;
    auto pages_of = [&](int64_t tokens) { return (tokens + v.page_tokens - 1) >> v.page_shift; };
    std::deque<Live> waiting;
    {
        const int32_t* p = prompts;
        for (int i = 0; i < n_requests; p += requests[i].n_prompt, i++) {
            const tsb_serve_request& r = requests[i];
            TSB_REQUIRE(ctx, r.n_prompt > 0 && r.max_new_tokens > 0 && r.max_new_tokens <= out_stride, "request %d: empty prompt, or a budget outside 1..%d", i, out_stride);
            const int64_t most = (int64_t)r.n_prompt + r.max_new_tokens;
            if (most > max_ctx || pages_of(most) > v.max_pages_per_seq || pages_of(most) > v.num_pages)
                return tsb_fail(ctx, TSB_ERR_INVALID, "request %d: %lld positions exceed the context window %d or the pool", i, (long long)most, max_ctx);
            Live l;
            l.request = i, l.prompt = p, l.n_prompt = r.n_prompt, l.budget = r.max_new_tokens;
            waiting.push_back(l);
            out_counts[i] = 0, out_reasons[i] = 0;
        }
    }
    std::vector<int> free_streams;
    for (int q = s->n_streams - 1; q >= 0; q--) {
        if ((rc = tsb_producer_reset(s, q))) return rc;
        free_streams.push_back(q);
    }
    std::vector<Live> live;
    tsb_serve_stats st{};
    const double t0 = now_s();
    auto fail = [&](int32_t code) {  // a failed run leaves no stream occupied
        const std::string why = ctx->last_error;
        for (const Live& l : live) tsb_producer_reset(s, l.stream);
        ctx->last_error = why;
        return code;
    };
    std::vector<RowGroup> groups;
    std::vector<int32_t> feed, want, tokens;
    std::vector<const Live*> who;
    while (!waiting.empty() || !live.empty()) {
        while (!waiting.empty() && !free_streams.empty() &&
               pages_of((int64_t)waiting.front().n_prompt + waiting.front().budget) <= (int64_t)rt.kv->free_pages.size()) {
            Live l = waiting.front();
            l.stream = free_streams.back();
            if ((rc = tsb_kv_reserve(rt.kv, l.stream, (int64_t)l.n_prompt + l.budget))) return fail(rc);
            waiting.pop_front(), free_streams.pop_back();
            live.push_back(l);
        }
        st.most_live = std::max(st.most_live, (int32_t)live.size());
        groups.clear(), feed.clear(), want.clear(), who.clear();
        auto take = [&](const Live& l, const int32_t* toks, int n, bool logits) {
            groups.push_back({l.stream, (int)feed.size(), n, tsb_kv_cursor(rt.kv, l.stream)});
            feed.insert(feed.end(), toks, toks + n);
            if (logits) want.push_back((int32_t)feed.size() - 1), who.push_back(&l);
        };
        for (Live& l : live)
            if (l.fed == l.n_prompt) take(l, &l.next, 1, true), st.decode_rows++;
        for (Live& l : live) {
            const int n = std::min(std::min(prefill_chunk, l.n_prompt - l.fed), s->pass_rows - (int)feed.size());
            if (l.fed == l.n_prompt || n <= 0) continue;
            take(l, l.prompt + l.fed, n, l.fed + n == l.n_prompt);
            l.fed += n, st.prompt_rows += n;
        }
        if ((rc = session_ragged_pass(s, groups.data(), (int)groups.size(), feed.data(), (int)feed.size(), want.data(), (int)want.size()))) return fail(rc);
        st.steps++, st.rows += (int64_t)feed.size();
        if (who.empty()) continue;
        if ((rc = sample_rows(s, who, cfg, tokens))) return fail(rc);
        for (size_t i = 0; i < who.size(); i++) {
            Live& l = const_cast<Live&>(*who[i]);
            l.next = tokens[i];
            out_tokens[(size_t)l.request * out_stride + l.generated++] = l.next;
            out_counts[l.request] = l.generated;
            bool stop = false;
            for (int k = 0; k < cfg->n_stop && k < 8; k++) stop |= cfg->stop_tokens[k] == l.next;
            if (stop || l.generated >= l.budget) {
                out_reasons[l.request] = stop ? 1 : 0;
                if ((rc = tsb_producer_reset(s, l.stream))) return fail(rc);
                free_streams.push_back(l.stream);
                l.request = -1;
            }
        }
        live.erase(std::remove_if(live.begin(), live.end(), [](const Live& l) { return l.request < 0; }), live.end());
    }
    st.seconds = now_s() - t0;
    if (stats) *stats = st;
    return TSB_OK;
}
