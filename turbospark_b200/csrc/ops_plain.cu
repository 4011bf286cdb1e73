// The mechanisms of output-norm and pre-norm layers as operators (include/tsb.h).
#include "gemm_plain.cuh"
#include "recurrence.cuh"
#include "rowops_plain.cuh"
#include "scan.cuh"
#include "sublayer.cuh"

namespace {

bool power_of_two(int n) { return n > 0 && (n & (n - 1)) == 0; }
bool known(int32_t type) { return type == TSB_BF16 || type == TSB_F32; }

int32_t check_portions(tsb_ctx* ctx, const tsb_row_desc* rows_dev, int32_t rows, int32_t rows_per_seq) {
    TSB_REQUIRE(ctx, rows_dev && rows > 0 && rows_per_seq > 0 && rows % rows_per_seq == 0, "rows must be whole portions of rows_per_seq");
    return TSB_OK;
}
int32_t ring_of(tsb_ctx* ctx, float* state, float* before, int32_t width, int32_t taps, int32_t n_streams, int32_t ring, int32_t rows_per_seq, RowRing& out, bool& use_before) {
    out.ring = state, out.before = before, out.width = width, out.ring_rows = ring, out.keep = taps > 1 ? taps - 1 : 0, out.n_streams = n_streams;
    use_before = out.keep > 0 && rows_per_seq + out.keep > ring;
    TSB_REQUIRE(ctx, n_streams > 0, "a convolution has streams");
    TSB_REQUIRE(ctx, out.keep == 0 || (state && power_of_two(ring) && (!use_before || before)),
                "a convolution needs its state, ring a power of two, and the rows before portions longer than it");
    return TSB_OK;
}
ExpertLists lists_of(const tsb_expert_lists& l) {
    ExpertLists x;
    x.ids = l.ids, x.weight = l.weight, x.slot_of = l.slot_of, x.token_of = l.token_of, x.first = l.first;
    x.chunks = reinterpret_cast<ExpertChunk*>(l.chunks), x.n_chunks = l.n_chunks;
    return x;
}

}  // namespace

extern "C" {

int32_t tsb_output_norm_rows(tsb_ctx* ctx, tsb_stream s, int32_t type, const float* x_in, const float* y, int32_t d, const float* weight, int32_t groups, float eps,
                             const float* taps_w, int32_t taps, float* state, float* before, int32_t n_streams, int32_t ring, const tsb_row_desc* rows_dev, int32_t rows,
                             int32_t rows_per_seq, float* x_out, void* out, int64_t out_stride) {
    if (!ctx) return TSB_ERR_INVALID;
    int32_t rc = check_portions(ctx, rows_dev, rows, rows_per_seq);
    if (rc) return rc;
    TSB_REQUIRE(ctx, known(type) && x_in && y && weight && x_out && x_in != x_out && d > 0 && (taps == 0 || (taps_w && out && out_stride >= d)), "bad arguments");
    TSB_REQUIRE(ctx, sublayer_end_supported(d, groups, taps), "width %d in %d groups with %d taps is outside the kernels", d, groups, taps);
    TSB_REQUIRE(ctx, (uintptr_t)x_in % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)weight % 16 == 0 && (uintptr_t)taps_w % 16 == 0 && (uintptr_t)x_out % 16 == 0 &&
                         (uintptr_t)out % 16 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)before % 16 == 0, "buffers must be 16-byte aligned");
    SublayerEnd e;
    if ((rc = ring_of(ctx, state, before, d, taps, n_streams, ring, rows_per_seq, e.ring, e.use_before))) return rc;
    DeviceGuard g(ctx);
    e.x_in = x_in, e.x_out = x_out, e.d = d, e.y = y, e.norm_w = weight, e.groups = groups, e.eps = eps, e.taps_w = taps_w, e.taps = taps, e.out = out;
    e.out_stride = out_stride, e.rows = rows_dev, e.n_rows = rows, e.tiles = RowTiles::uniform(rows, rows_per_seq, sublayer_rows_per_tile(ctx, rows));
    TSB_CUDA(ctx, launch_sublayer_end(ctx, (cudaStream_t)s, type == TSB_F32, e));
    return TSB_OK;
}

int32_t tsb_projection_norm_rows(tsb_ctx* ctx, tsb_stream s, tsb_kv* cache, int32_t layer, const float* raw, int64_t raw_stride, int32_t n_q, int32_t n_k, int32_t width,
                                 const float* q_weight, const float* k_weight, float eps, const tsb_row_desc* rows_dev, int32_t rows, void* q, int64_t q_stride) {
    if (!ctx || !cache) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, !cache->key_layers.empty() && layer >= 0 && layer < (int)cache->key_layers.size(), "a plain cache and one of its layers expected");
    const KeyView& kv = cache->key_layers[layer];
    TSB_REQUIRE(ctx, raw && rows_dev && rows > 0 && n_q > 0 && n_k > 0 && n_k <= kv.kv_heads && width > 0 && width <= kv.head_dim && q && q_weight && k_weight &&
                         raw_stride >= (int64_t)(n_q + n_k) * width && q_stride >= (int64_t)n_q * kv.head_dim, "bad arguments");
    DeviceGuard g(ctx);
    ProjectionNorms p;
    p.raw = raw, p.raw_stride = raw_stride, p.n_q = n_q, p.n_k = n_k, p.width = width, p.q_weight = q_weight, p.k_weight = k_weight, p.eps = eps, p.q = q;
    p.q_stride = q_stride, p.q_step = kv.head_dim, p.keys = kv, p.rows = rows_dev;
    TSB_CUDA(ctx, launch_projection_norms(ctx, (cudaStream_t)s, kv.elem_bytes == 4, p, rows));
    return TSB_OK;
}

int32_t tsb_short_conv_rows(tsb_ctx* ctx, tsb_stream s, int32_t type, const void* in, int64_t in_stride, int32_t channels, const float* taps_w, int32_t taps,
                            const float* bias, float* state, float* before, int32_t n_streams, int32_t ring, const tsb_row_desc* rows_dev, int32_t rows,
                            int32_t rows_per_seq, void* out, int64_t out_stride) {
    if (!ctx) return TSB_ERR_INVALID;
    int32_t rc = check_portions(ctx, rows_dev, rows, rows_per_seq);
    if (rc) return rc;
    TSB_REQUIRE(ctx, known(type) && in && out && taps_w && bias && channels > 0 && taps > 0 && taps <= CONV_MAX_TAPS && in_stride >= channels && out_stride >= channels,
                "bad arguments");
    ShortConv c;
    if ((rc = ring_of(ctx, state, before, channels, taps, n_streams, ring, rows_per_seq, c.ring, c.use_before))) return rc;
    DeviceGuard g(ctx);
    c.in = in, c.in_stride = in_stride, c.out = out, c.out_stride = out_stride, c.channels = channels, c.taps = taps, c.w = taps_w, c.bias = bias, c.rows = rows_dev;
    c.n_rows = rows, c.tiles = RowTiles::uniform(rows, rows_per_seq, sublayer_rows_per_tile(ctx, rows));
    TSB_CUDA(ctx, launch_short_conv(ctx, (cudaStream_t)s, type == TSB_F32, c));
    return TSB_OK;
}

int32_t tsb_recurrence_rows(tsb_ctx* ctx, tsb_stream s, int32_t type, const tsb_recurrence* r, const tsb_row_desc* rows_dev, int32_t rows, int32_t rows_per_seq,
                            int32_t chunked) {
    if (!ctx || !r) return TSB_ERR_INVALID;
    int32_t rc = check_portions(ctx, rows_dev, rows, rows_per_seq);
    if (rc) return rc;
    const int per_key = r->heads_per_key > 0 ? r->heads_per_key : 1;
    const bool forget = r->kind == TSB_REC_FORGET, mlstm = r->kind == TSB_REC_MLSTM, ssd = r->kind == TSB_REC_SSD;
    TSB_REQUIRE(ctx, known(type) && (forget || mlstm || ssd) && r->heads > 0 && r->dim > 0 && r->dim <= REC_MAX_DIM && r->vdim > 0 && r->heads % per_key == 0, "bad recurrence");
    TSB_REQUIRE(ctx, r->q && (forget || r->k) && r->v && r->gate && r->out && r->state && (!forget || r->lower) && (!ssd || (r->a_log && r->skip)) &&
                         (!mlstm || (r->norm && r->top && r->cap > 0.f)), "a buffer is missing");
    TSB_REQUIRE(ctx, power_of_two(r->ring) && r->ring > 1 && r->n_streams > 0 && (uintptr_t)r->state % 16 == 0, "ring is a power of two above one");
    TSB_REQUIRE(ctx, !chunked || (type == TSB_BF16 && recurrence_chunks_supported(r->kind, r->dim, r->vdim)), "no chunked kernel for this type and these sizes");
    TSB_REQUIRE(ctx, !chunked || ((uintptr_t)r->q % 16 == 0 && (uintptr_t)r->k % 16 == 0 && (uintptr_t)r->v % 16 == 0 && (uintptr_t)r->out % 8 == 0 && r->q_stride % 8 == 0 &&
                                  r->k_stride % 8 == 0 && r->v_stride % 8 == 0 && r->out_stride % 2 == 0 && r->scratch && (uintptr_t)r->scratch % 16 == 0 &&
                                  (!forget || ((uintptr_t)r->gate % 16 == 0 && r->gate_stride % 4 == 0))), "rows start on 16-byte boundaries, and there is scratch memory");
    DeviceGuard g(ctx);
    Recurrence x;
    x.kind = r->kind, x.heads = r->heads, x.dim = r->dim, x.vdim = r->vdim, x.heads_per_key = per_key, x.q = r->q, x.k = r->k, x.v = r->v;
    x.q_stride = r->q_stride, x.k_stride = r->k_stride, x.v_stride = r->v_stride, x.gate = r->gate, x.gate_stride = r->gate_stride, x.lower = r->lower;
    x.a_log = r->a_log, x.skip = r->skip, x.cap = r->cap, x.q_scale = r->q_scale == 0.f ? 1.f : r->q_scale, x.out = r->out, x.out_stride = r->out_stride;
    x.state.s = r->state, x.state.norm = r->norm, x.state.top = r->top, x.state.ring = r->ring, x.state.n_streams = r->n_streams, x.rows = rows_dev, x.n_rows = rows;
    const RowTiles portions = RowTiles::uniform(rows, rows_per_seq, rows_per_seq);
    RecurrenceChunks c;
    c.chunks = RowTiles::uniform(rows, rows_per_seq, REC_CHUNK), c.n_portions = rows / rows_per_seq, c.rows_per_seq = rows_per_seq, c.scratch = r->scratch;
    TSB_CUDA(ctx, chunked ? launch_recurrence_chunks(ctx, (cudaStream_t)s, x, c) : launch_recurrence_rows(ctx, (cudaStream_t)s, type == TSB_F32, x, portions));
    return TSB_OK;
}

size_t tsb_recurrence_scratch_bytes(int32_t kind, int32_t heads, int32_t dim, int32_t vdim, int32_t rows, int32_t rows_per_seq) {
    if (heads <= 0 || dim <= 0 || vdim <= 0 || rows <= 0 || rows_per_seq <= 0) return 0;
    return recurrence_scratch_bytes(kind, heads, dim, vdim, rows / rows_per_seq * ((rows_per_seq + REC_CHUNK - 1) / REC_CHUNK));
}

int32_t tsb_gated_norm_rows(tsb_ctx* ctx, tsb_stream s, int32_t type, const float* o, int64_t o_stride, int32_t width, int32_t groups, const float* weight, int32_t weight_n,
                            float eps, float scale, const void* pre_gate, const void* post_gate, int64_t gate_stride, int32_t rows, void* out, int64_t out_stride) {
    if (!ctx) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, known(type) && o && weight && out && rows > 0 && width > 0 && width <= 24 * 1024 && groups > 0 && width % groups == 0 && weight_n > 0 &&
                         o_stride >= width && out_stride >= width && ((!pre_gate && !post_gate) || gate_stride >= width), "bad arguments");
    TSB_REQUIRE(ctx, (uintptr_t)o % 16 == 0 && (uintptr_t)weight % 16 == 0, "o and weight must be 16-byte aligned");
    DeviceGuard g(ctx);
    GatedNorm n;
    n.o = o, n.o_stride = o_stride, n.width = width, n.groups = groups, n.weight = weight, n.weight_n = weight_n, n.eps = eps, n.scale = scale, n.pre_gate = pre_gate;
    n.post_gate = post_gate, n.gate_stride = gate_stride, n.out = out, n.out_stride = out_stride;
    TSB_CUDA(ctx, launch_gated_norm(ctx, (cudaStream_t)s, type == TSB_F32, n, rows));
    return TSB_OK;
}

int32_t tsb_route_experts(tsb_ctx* ctx, tsb_stream s, const float* logits, const float* correction, int32_t experts, int32_t top, int32_t groups, int32_t keep, int32_t rows,
                          int32_t chunk_slots, const tsb_expert_lists* lists) {
    if (!ctx || !lists) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, logits && correction && rows > 0 && chunk_slots >= 8 && routing_supported(experts, top, groups, keep), "bad arguments");
    TSB_REQUIRE(ctx, lists->ids && lists->weight && lists->slot_of && lists->token_of && lists->first && lists->chunks && lists->n_chunks, "a list is missing");
    DeviceGuard g(ctx);
    ExpertRouting r;
    r.logits = logits, r.logits_stride = experts, r.correction = correction, r.experts = experts, r.top = top, r.groups = groups, r.keep = keep, r.rows = rows;
    r.chunk_slots = chunk_slots, r.lists = lists_of(*lists);
    TSB_CUDA(ctx, launch_route_experts(ctx, (cudaStream_t)s, r));
    return TSB_OK;
}

int32_t tsb_plain_gemm_experts(tsb_ctx* ctx, tsb_stream s, int32_t type, const void* w, int32_t experts, int64_t w_rows, int64_t cols, const void* x, int64_t x_stride,
                               int32_t x_rows, int32_t by_token, const tsb_expert_lists* lists, int32_t slots, int32_t chunk_slots, int32_t tensor, int32_t pairs, void* y,
                               int64_t y_stride, int32_t n_valid) {
    if (!ctx || !lists) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, known(type) && w && x && y && experts > 0 && experts <= EXPERTS_MAX && slots > 0 && lists->first && lists->token_of && lists->chunks && lists->n_chunks,
                "bad arguments");
    TSB_REQUIRE(ctx, w_rows > 0 && w_rows % PLAIN_ROW_PAD == 0 && cols > 0 && cols % PLAIN_COL_PAD == 0 && x_stride >= cols && x_stride % 8 == 0,
                "rows must be a multiple of %d and cols of %d", PLAIN_ROW_PAD, PLAIN_COL_PAD);
    TSB_REQUIRE(ctx, (uintptr_t)w % 16 == 0 && (uintptr_t)x % 16 == 0, "w and x must be 16-byte aligned");
    TSB_REQUIRE(ctx, n_valid > 0 && n_valid <= (pairs ? w_rows / 2 : w_rows) && y_stride >= n_valid, "bad output");
    TSB_REQUIRE(ctx, tensor ? type == TSB_BF16 && !by_token && x_rows >= 256 : chunk_slots == (type == TSB_F32 ? EXPERT_CHUNK_F32 : 8) ||
                         (type == TSB_BF16 && chunk_slots == EXPERT_CHUNK_FEW), "chunks or rows of x do not fit the kernel");
    DeviceGuard g(ctx);
    const ExpertLists l = lists_of(*lists);
    PlainExperts e;
    e.n = experts, e.slots = slots, e.first = l.first, e.token_of = by_token ? l.token_of : nullptr, e.chunks = l.chunks, e.n_chunks = l.n_chunks, e.chunk_slots = chunk_slots;
    PlainEpi p;
    p.kind = PLAIN_MIXER;
    if (pairs) p.pair_row0 = 0, p.n_pairs = n_valid, p.act = PLAIN_SILU, p.a = y, p.a_stride = y_stride;
    else p.n_seg = 1, p.seg[0].end = n_valid, p.seg[0].p = y, p.seg[0].stride = y_stride;
    TSB_CUDA(ctx, launch_plain_gemm_experts(ctx, (cudaStream_t)s, type == TSB_F32, tensor != 0, PlainMat{const_cast<void*>(w), w_rows, cols}, x, x_stride, x_rows, e, p));
    return TSB_OK;
}

int32_t tsb_pre_norm_rows(tsb_ctx* ctx, tsb_stream s, int32_t type, const float* x, int32_t d, const float* weight, float eps, int32_t rows, void* out,
                          int64_t out_stride) {
    if (!ctx) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, known(type) && x && weight && out && d > 0 && rows > 0 && out_stride >= d, "bad arguments");
    TSB_REQUIRE(ctx, (uintptr_t)x % 16 == 0 && (uintptr_t)weight % 16 == 0 && (uintptr_t)out % 16 == 0, "buffers must be 16-byte aligned");
    DeviceGuard g(ctx);
    TSB_CUDA(ctx, launch_pre_norm(ctx, (cudaStream_t)s, type == TSB_F32, x, d, weight, eps, rows, out, out_stride));
    return TSB_OK;
}

int32_t tsb_turned_norm_rows(tsb_ctx* ctx, tsb_stream s, tsb_kv* cache, int32_t layer, const tsb_turned_norms* n, const tsb_row_desc* rows_dev, int32_t rows) {
    if (!ctx || !cache || !n) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, !cache->key_layers.empty() && layer >= 0 && layer < (int)cache->key_layers.size(), "a plain cache and one of its layers expected");
    const KeyView& kv = cache->key_layers[layer];
    TSB_REQUIRE(ctx, n->raw && rows_dev && rows > 0 && n->n_q > 0 && n->n_k > 0 && n->n_k <= kv.kv_heads && n->width > 0 && n->width <= kv.head_dim && n->q && n->q_weight &&
                         n->k_weight && n->n_v >= 0 && n->n_v <= kv.kv_heads && n->raw_stride >= (int64_t)(n->n_q + n->n_k) * n->width + (int64_t)n->n_v * n->v_width &&
                         n->q_stride >= (int64_t)n->n_q * kv.head_dim, "bad arguments");
    TSB_REQUIRE(ctx, n->n_v == 0 || (!n->projection && n->v_width > 0 && kv.value_off > 0 && n->v_width <= kv.head_step - kv.value_off), "the cache has no room for the values");
    TSB_REQUIRE(ctx, (!n->rot || (n->rot_half > 0 && 2 * n->rot_half <= n->width)) && (!n->turn || (n->turn_half > 0 && 2 * n->turn_half <= n->v_width)), "more columns are turned than there are");
    const float2 *rot = reinterpret_cast<const float2*>(n->rot), *turn = reinterpret_cast<const float2*>(n->turn);
    DeviceGuard g(ctx);
    if (n->projection) {
        ProjectionNorms p;
        p.raw = n->raw, p.raw_stride = n->raw_stride, p.n_q = n->n_q, p.n_k = n->n_k, p.width = n->width, p.q_weight = n->q_weight, p.k_weight = n->k_weight, p.eps = n->eps;
        p.q = n->q, p.q_stride = n->q_stride, p.q_step = kv.head_dim, p.keys = kv, p.rows = rows_dev, p.rot = rot, p.rot_half = rot ? n->rot_half : 0;
        TSB_CUDA(ctx, launch_projection_norms(ctx, (cudaStream_t)s, kv.elem_bytes == 4, p, rows));
        return TSB_OK;
    }
    HeadNorms h;
    h.raw = n->raw, h.raw_stride = n->raw_stride, h.n_q = n->n_q, h.n_k = n->n_k, h.n_v = n->n_v, h.width = n->width, h.v_width = n->v_width, h.q_weight = n->q_weight;
    h.k_weight = n->k_weight, h.eps = n->eps, h.q = n->q, h.q_stride = n->q_stride, h.q_step = h.q_width = kv.head_dim, h.keys = kv, h.rows = rows_dev;
    h.rot = rot, h.rot_half = rot ? n->rot_half : 0, h.turn = turn, h.turn_half = turn ? n->turn_half : 0;
    TSB_CUDA(ctx, launch_head_norms(ctx, (cudaStream_t)s, kv.elem_bytes == 4, h, rows));
    return TSB_OK;
}

int32_t tsb_block_mean_rows(tsb_ctx* ctx, tsb_stream s, tsb_kv* cache, int32_t layer, const tsb_row_desc* rows_dev, int32_t rows) {
    if (!ctx || !cache) return TSB_ERR_INVALID;
    TSB_REQUIRE(ctx, layer >= 0 && layer < (int)cache->pool_sizes.size() && cache->pool_sizes[layer] > 0 && rows_dev && rows > 0, "a layer that keeps blocks expected");
    DeviceGuard g(ctx);
    BlockMeans b;
    b.keys = cache->key_layers[layer], b.pooled = cache->pooled_layers[layer], b.pool = cache->pool_sizes[layer], b.rows = rows_dev;
    TSB_CUDA(ctx, launch_block_means(ctx, (cudaStream_t)s, b.keys.elem_bytes == 4, b, rows));
    return TSB_OK;
}

int32_t tsb_gated_scan_rows(tsb_ctx* ctx, tsb_stream s, int32_t type, const float* gate, int64_t gate_stride, const void* out_gate, int64_t out_gate_stride, int32_t width,
                            float* state, int32_t n_streams, int32_t ring, const tsb_row_desc* rows_dev, int32_t rows, int32_t rows_per_seq, int32_t chunked, void* sums, void* out, int64_t out_stride) {
    if (!ctx) return TSB_ERR_INVALID;
    int32_t rc = check_portions(ctx, rows_dev, rows, rows_per_seq);
    if (rc) return rc;
    TSB_REQUIRE(ctx, !chunked || rows_per_seq <= SCAN_CHUNK || (sums && (uintptr_t)sums % 8 == 0), "portions of several chunks need room for their sums");
    TSB_REQUIRE(ctx, known(type) && gate && out_gate && state && out && width > 0 && gate_stride >= 2 * (int64_t)width && out_gate_stride >= width && out_stride >= width, "bad arguments");
    TSB_REQUIRE(ctx, power_of_two(ring) && ring > 1 && n_streams > 0, "ring is a power of two above one");
    DeviceGuard g(ctx);
    GatedScan x;
    x.gate = gate, x.gate_stride = gate_stride, x.out_gate = out_gate, x.out_gate_stride = out_gate_stride, x.out = out, x.out_stride = out_stride, x.width = width;
    x.state.s = state, x.state.ring = ring, x.state.n_streams = n_streams, x.rows = rows_dev;
    x.n_rows = rows;
    const bool f32 = type == TSB_F32;
    TSB_CUDA(ctx, chunked ? launch_gated_scan_chunks(ctx, (cudaStream_t)s, f32, x, RowTiles::uniform(rows, rows_per_seq, SCAN_CHUNK), rows_per_seq > SCAN_CHUNK, static_cast<float2*>(sums))
                          : launch_gated_scan_rows(ctx, (cudaStream_t)s, f32, x, RowTiles::uniform(rows, rows_per_seq, rows_per_seq)));
    return TSB_OK;
}

}  // extern "C"
