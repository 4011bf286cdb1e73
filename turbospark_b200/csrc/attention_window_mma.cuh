// The mma.sync attention kernels over a plain paged cache (attention_window.cu describes them).  Instantiated once for
// caches whose values are their keys (KV = false: a key tile serves both products) and once for caches with values of their own
// (KV = true: a stage of the ring holds a key tile and a value tile).  PRE: the prefix before the window goes first, in key tiles of its own;
// its rows are counted from zero, and a query sees those below its own number of them.
#pragma once
#include "attention_window_dev.cuh"
#include "mma_dev.cuh"

namespace {

constexpr int TOK = 64;   // tokens per key tile
// key tiles in flight
template <int D, bool KV>
constexpr int ring_stages() { return KV && D > 128 ? 2 : 3; }

template <int D>
struct Geo {
    static constexpr int PITCH = D <= 32 ? 64 : D <= 64 ? 128 : D <= 128 ? 256 : 512;  // bytes of a row in shared memory
    static constexpr int CH = D / 8;                                                  // 16-byte chunks of a row
    // byte offset of chunk c of row r: the chunks of a row are permuted so that eight rows' worth of one chunk spread over
    // all banks
    static __device__ __forceinline__ uint32_t off(int r, int c) {
        return (uint32_t)(r * PITCH + ((D <= 32 ? (c ^ ((r >> 1) & 3)) : (c ^ (r & 7))) << 4));
    }
};

// Raw scores of an mma accumulator tile -> base-2 logits with cap, bias and mask, and the lane's running maximum per query.
// KEYS_M: rows of the tile are keys (16 per n) and columns queries; else rows are queries and columns keys (8 per n).
// db[h]: distance of the lane's first key from its query h; span[h]: the distance from which on the query sees nothing.  A linear bias has its
// slope, times log2(e), in r1.
template <int N, bool KEYS_M>
__device__ __forceinline__ void base2_logits(float (&s)[N][4], const WindowAttn& a, const ScoreConst& sc, const float (&db)[2], const float (&r1)[2],
                                             const float (&r2)[2], const float (&span)[2], bool edge, float (&mx)[2]) {
    if (a.cap > 0.f) {
        float big = 0.f;
#pragma unroll
        for (int n = 0; n < N; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) big = fmaxf(big, fabsf(s[n][i]));
        if (__any_sync(0xffffffffu, big > sc.small)) {
#pragma unroll
            for (int n = 0; n < N; n++)
#pragma unroll
                for (int i = 0; i < 4; i++) s[n][i] = fmaf(-2.f * sc.c_out, rcp(ex2(s[n][i] * sc.s_in) + 1.f), sc.c_out);  // tanh(y) = 1 - 2 / (e^(2y) + 1)
        } else {
#pragma unroll
            for (int n = 0; n < N; n++)
#pragma unroll
                for (int i = 0; i < 4; i += 2) {
                    const float2 x = make_float2(s[n][i], s[n][i + 1]), v = mul2(x, sc.factor(x));
                    s[n][i] = v.x, s[n][i + 1] = v.y;
                }
        }
    } else {
#pragma unroll
        for (int n = 0; n < N; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) s[n][i] *= sc.s_in;
    }
#pragma unroll
    for (int n = 0; n < N; n++)
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int h = KEYS_M ? i & 1 : i >> 1;
            const float dist = db[h] - (float)(KEYS_M ? n * 16 + (i >> 1) * 8 : n * 8 + (i & 1));
            if (a.r1) s[n][i] = fmaf(-r1[h], lg2(fmaf(r2[h], dist, 1.f)), s[n][i]);
            if (a.slopes) s[n][i] = fmaf(-r1[h], dist, s[n][i]);
            if (edge && (dist < 0.f || dist >= span[h])) s[n][i] = -INFINITY;
            mx[h] = fmaxf(mx[h], s[n][i]);
        }
}

// The SL warps that shared a query tile's tokens have left (m, l) and O per query in shared memory, wo[slice][QT][D + 4] and
// wml[slice][QT].  One run: the finished rows are written.  Several runs (TICKET): the run's share goes to memory and the
// last run of the tile to finish adds all of them, in order; without TICKET a merge launch does.
template <int D, int QT, int SL, int NTHR, bool TICKET>
__device__ __forceinline__ void finish_slices(const WindowAttn& a, int row_first, int kvh, int grp, int n_queries, int n_splits, const float* wo,
                                              const float2* wml, float* __restrict__ part_o, float2* __restrict__ part_ml, uint32_t* __restrict__ tickets) {
    constexpr int DP = D + 4;
    __shared__ uint32_t s_ticket;
    const int64_t tile_id = (int64_t)blockIdx.z * a.keys.kv_heads + kvh;
    const int64_t share = (tile_id * n_splits + blockIdx.x) * QT;
    auto store = [&](int qi, int c, float4 v, float m, float l) {
        const int row = row_first + qi / grp, head = kvh * grp + qi % grp;
        const float f = head_factor(a, row, head, m, l);
        if (a.turn) turn_back(a, row, c, v.x, v.y), turn_back(a, row, c + 2, v.z, v.w);
        if (a.value_gate) value_gates(a, row, head, c, v);
        *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(a.out) + (int64_t)row * a.out_stride + head * D + c) =
            make_uint2(pack_bf16(v.x * f, v.y * f), pack_bf16(v.z * f, v.w * f));
    };
    for (int i = threadIdx.x; i < n_queries * (D / 4); i += NTHR) {
        const int qi = i / (D / 4), c = (i % (D / 4)) * 4;
        float m = -INFINITY, l = 0.f;
#pragma unroll
        for (int k = 0; k < SL; k++) m = fmaxf(m, wml[k * QT + qi].x);
        const float mu = m == -INFINITY ? 0.f : m;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int k = 0; k < SL; k++) {
            const float2 v = wml[k * QT + qi];
            const float f = ex2(v.x - mu);
            l = fmaf(v.y, f, l);
            const float4 x = *reinterpret_cast<const float4*>(wo + (size_t)(k * QT + qi) * DP + c);
            acc.x = fmaf(x.x, f, acc.x), acc.y = fmaf(x.y, f, acc.y), acc.z = fmaf(x.z, f, acc.z), acc.w = fmaf(x.w, f, acc.w);
        }
        if (n_splits == 1) {
            store(qi, c, acc, m, l);
        } else {
            *reinterpret_cast<float4*>(part_o + (share + qi) * D + c) = acc;
            if (c == 0) part_ml[share + qi] = make_float2(m, l);
        }
    }
    if (!TICKET || n_splits == 1) return;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        s_ticket = atomicAdd(&tickets[tile_id], 1u);
        if (s_ticket == (uint32_t)n_splits - 1) tickets[tile_id] = 0;
    }
    __syncthreads();
    if (s_ticket != (uint32_t)n_splits - 1) return;
    __threadfence();
    const int64_t first = tile_id * n_splits * QT;
    for (int i = threadIdx.x; i < n_queries * (D / 4); i += NTHR) {
        const int qi = i / (D / 4), c = (i % (D / 4)) * 4;
        float m = -INFINITY, l = 0.f;
#pragma unroll 8
        for (int k = 0; k < n_splits; k++) m = fmaxf(m, __ldcg(&part_ml[first + k * QT + qi]).x);
        const float mu = m == -INFINITY ? 0.f : m;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int k = 0; k < n_splits; k++) {
            const float2 v = __ldcg(&part_ml[first + k * QT + qi]);
            const float4 x = __ldcg(reinterpret_cast<const float4*>(part_o + (first + k * QT + qi) * D + c));
            const float f = ex2(v.x - mu);
            l = fmaf(v.y, f, l);
            acc.x = fmaf(x.x, f, acc.x), acc.y = fmaf(x.y, f, acc.y), acc.z = fmaf(x.z, f, acc.z), acc.w = fmaf(x.w, f, acc.w);
        }
        store(qi, c, acc, m, l);
    }
}

template <int D, int MT, int SL, bool KV>
constexpr size_t wattn_smem() {
    const size_t ring = (size_t)ring_stages<D, KV>() * TOK * Geo<D>::PITCH * (KV ? 2 : 1) + (SL == 1 ? (size_t)MT * 16 * Geo<D>::PITCH : 0);
    const size_t merge = SL > 1 ? (size_t)MT * SL * 16 * ((D + 4) * 4 + 8) : 0;
    return ring > merge ? ring : merge;
}

template <int D, int MT, int SL, bool KV, bool PRE>
__global__ void __launch_bounds__(32 * MT * SL, MT * SL <= 4 ? 3 : 1)
    window_attn_kernel(const __grid_constant__ WindowAttn a, const AttnTile* __restrict__ tiles, int tiles_per_group, int rows_per_seq, int rows_per_tile,
                       float* __restrict__ part_o, float2* __restrict__ part_ml, uint32_t* __restrict__ tickets, uint32_t* __restrict__ err) {
    using G = Geo<D>;
    constexpr int KS = D / 16, NO = D / 8, QT = 16 * MT, NTHR = 32 * MT * SL;
    constexpr int WTOK = TOK / SL, NT8 = WTOK / 8, KK = WTOK / 16;
    constexpr int NST = ring_stages<D, KV>(), STAGE = TOK * G::PITCH * (KV ? 2 : 1), V_AT = KV ? TOK * G::PITCH : 0;
    constexpr bool QREG = SL > 1 ? D <= 128 : D <= 64;  // query fragments stay in registers
    extern __shared__ __align__(128) uint8_t smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int mt = warp % MT, sl = warp / MT;
    const int kvh = blockIdx.y, n_splits = gridDim.x;
    const int grp = a.n_q_heads / a.keys.kv_heads;

    int row_first, n_rows;
    if (tiles) {
        row_first = tiles[blockIdx.z].row_first, n_rows = tiles[blockIdx.z].n_rows;
    } else {
        const int in_group = ((int)blockIdx.z % tiles_per_group) * rows_per_tile;
        row_first = ((int)blockIdx.z / tiles_per_group) * rows_per_seq + in_group;
        n_rows = min(rows_per_tile, rows_per_seq - in_group);
    }
    const tsb_row_desc rd0 = a.rows[row_first];
    const int seq = rd0.seq, pos0 = rd0.base + rd0.slot;
    const int n_queries = n_rows * grp;
    if (seq < 0 || seq >= a.keys.max_seqs || n_queries > QT) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        pdl_wait();
        return;
    }
    // visible positions of the tile's queries, in whole key tiles; this CTA's run of them
    const int lo = first_visible(a, pos0) & ~(TOK - 1);
    const int hi = pos0 + n_rows, lo_last = first_visible(a, hi - 1);
    const int n_pre = PRE ? prefix_len(a, hi - 1) : 0, pre_all = PRE ? prefix_len(a, pos0) : 0;  // of the prefix: seen by some row, by every row
    const int pre_tiles = (n_pre + TOK - 1) / TOK;
    const int total = pre_tiles + (hi - lo + TOK - 1) / TOK;
    const int per = (total + n_splits - 1) / n_splits;
    const int t_first = min(total, (int)blockIdx.x * per), n_tiles = min(total, t_first + per) - t_first;
    const int begin = lo + (t_first - pre_tiles) * TOK;

    const uint32_t ring = smem_u32(smem);
    auto issue = [&](int tile, int stage) {
        constexpr int TPR = NTHR / TOK;  // threads per token row
        const int r = threadIdx.x / TPR, part = threadIdx.x % TPR;
        const bool pre = PRE && t_first + tile < pre_tiles;
        const int pos = (pre ? (t_first + tile) * TOK : begin + tile * TOK) + r;
        const __nv_bfloat16* src = pos >= (pre ? n_pre : hi) ? nullptr : PRE ? run_row(a, pre, seq, pos) : key_row<__nv_bfloat16>(a.keys, seq, pos);
        const bool ok = src != nullptr;
        src = ok ? src + (int64_t)kvh * a.keys.head_step : reinterpret_cast<const __nv_bfloat16*>(a.keys.base);
        const uint32_t dst = ring + stage * STAGE;
#pragma unroll
        for (int c = part; c < G::CH; c += TPR) cp16(dst + G::off(r, c), ok ? src + c * 8 : src, ok);
        if (KV) {
#pragma unroll
            for (int c = part; c < G::CH; c += TPR) cp16(dst + V_AT + G::off(r, c), ok ? src + a.keys.value_off + c * 8 : src, ok);
        }
        cp_async_commit();
    };
    auto prologue = [&]() {
#pragma unroll
        for (int i = 0; i < NST; i++) {
            if (i < n_tiles) issue(i, i);
            else cp_async_commit();
        }
    };
    // key tiles of earlier passes may start moving while the kernel that writes this pass's rows still runs
    // (a prefix: rows of positions before this pass)
    const bool early = begin + NST * TOK <= rd0.base && (!PRE || min(n_pre, (t_first + NST) * TOK) * max(a.pool, 1) <= rd0.base);
    if (early) prologue();
    pdl_wait();
    if (!early) prologue();

    // the lane's two queries: rows gid and gid + 8 of its m-tile
    const __nv_bfloat16* qp[2];
    int pq[2];
    float r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f}, span[2];
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int qi = mt * 16 + gid + 8 * h;
        const bool v = qi < n_queries;
        const int row = v ? qi / grp : 0, head = kvh * grp + (v ? qi % grp : 0);
        pq[h] = pos0 + row;  // an empty slot repeats the first query and is not stored
        qp[h] = reinterpret_cast<const __nv_bfloat16*>(a.q) + (int64_t)(row_first + row) * a.q_stride + head * D;
        if (a.r1) r1[h] = a.r1[head], r2[h] = a.r2[head];
        if (a.slopes) r1[h] = a.slopes[head] * 1.4426950408889634f;
        span[h] = visible_span(a, pq[h]);
    }
    uint32_t qa[QREG ? KS : 1][4];
    const uint32_t q_smem = ring + NST * STAGE;
    if (QREG) {
#pragma unroll
        for (int ks = 0; ks < (QREG ? KS : 0); ks++) {
            qa[ks][0] = *reinterpret_cast<const uint32_t*>(qp[0] + 16 * ks + 2 * tig);
            qa[ks][1] = *reinterpret_cast<const uint32_t*>(qp[1] + 16 * ks + 2 * tig);
            qa[ks][2] = *reinterpret_cast<const uint32_t*>(qp[0] + 16 * ks + 8 + 2 * tig);
            qa[ks][3] = *reinterpret_cast<const uint32_t*>(qp[1] + 16 * ks + 8 + 2 * tig);
        }
    } else if (SL == 1) {
        for (int i = threadIdx.x; i < QT * G::CH; i += NTHR) {
            const int qi = i / G::CH, c = i % G::CH;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (qi < n_queries)
                v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(a.q) + (int64_t)(row_first + qi / grp) * a.q_stride +
                                                    (kvh * grp + qi % grp) * D + c * 8);
            *reinterpret_cast<uint4*>(smem + NST * STAGE + G::off(qi, c)) = v;
        }
    }

    const ScoreConst sc(a);

    float o[NO][4];
#pragma unroll
    for (int n = 0; n < NO; n++)
#pragma unroll
        for (int i = 0; i < 4; i++) o[n][i] = 0.f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

    for (int tile = 0; tile < n_tiles; tile++) {
        const int stage = tile % NST;
        cp_async_wait<NST - 1>();
        __syncthreads();
        const uint32_t kt = ring + stage * STAGE, vt = kt + V_AT;
        const int tok0 = sl * WTOK;
        const bool pre = PRE && t_first + tile < pre_tiles;
        const int p0 = (pre ? (t_first + tile) * TOK : begin + tile * TOK) + tok0;
        float s[NT8][4];
#pragma unroll
        for (int n = 0; n < NT8; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) s[n][i] = 0.f;
#pragma unroll
        for (int kp = 0; kp < KS / 2; kp++) {
            uint32_t a0[4], a1[4];
            if (QREG) {
#pragma unroll
                for (int i = 0; i < 4; i++) a0[i] = qa[QREG ? 2 * kp : 0][i], a1[i] = qa[QREG ? 2 * kp + 1 : 0][i];
            } else if (SL == 1) {
                const int r = mt * 16 + (lane & 15), c = kp * 4 + (lane >> 4);
                ldsm4(a0, q_smem + G::off(r, c));
                ldsm4(a1, q_smem + G::off(r, c + 2));
            } else {
                a0[0] = *reinterpret_cast<const uint32_t*>(qp[0] + 32 * kp + 2 * tig), a0[1] = *reinterpret_cast<const uint32_t*>(qp[1] + 32 * kp + 2 * tig);
                a0[2] = *reinterpret_cast<const uint32_t*>(qp[0] + 32 * kp + 8 + 2 * tig), a0[3] = *reinterpret_cast<const uint32_t*>(qp[1] + 32 * kp + 8 + 2 * tig);
                a1[0] = *reinterpret_cast<const uint32_t*>(qp[0] + 32 * kp + 16 + 2 * tig), a1[1] = *reinterpret_cast<const uint32_t*>(qp[1] + 32 * kp + 16 + 2 * tig);
                a1[2] = *reinterpret_cast<const uint32_t*>(qp[0] + 32 * kp + 24 + 2 * tig), a1[3] = *reinterpret_cast<const uint32_t*>(qp[1] + 32 * kp + 24 + 2 * tig);
            }
#pragma unroll
            for (int n = 0; n < NT8; n++) {
                uint32_t b[4];
                ldsm4(b, kt + G::off(tok0 + n * 8 + (lane & 7), kp * 4 + (lane >> 3)));
                mma_bf16(s[n], a0, b[0], b[1]);
                mma_bf16(s[n], a1, b[2], b[3]);
            }
        }
        // the mask only where the tile meets an edge
        const bool edge = pre ? p0 + WTOK > pre_all : p0 + WTOK > pos0 || p0 < lo_last;
        float mx[2] = {-INFINITY, -INFINITY}, db[2], sp[2];
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int last = pre ? prefix_len(a, pq[h]) - 1 : pq[h];  // the last one that the query sees
            db[h] = (float)(last - p0 - 2 * tig), sp[h] = pre ? 3e38f : span[h];
        }
        base2_logits<NT8, false>(s, a, sc, db, r1, r2, sp, edge, mx);
        float alpha[2], m_use[2];
#pragma unroll
        for (int h = 0; h < 2; h++) {
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
            const float m_new = fmaxf(m_run[h], mx[h]);
            m_use[h] = m_new == -INFINITY ? 0.f : m_new;
            alpha[h] = ex2(m_run[h] - m_use[h]);  // 0 while nothing was visible
            m_run[h] = m_new;
        }
        float rs[2] = {0.f, 0.f};
        uint32_t pa[KK][4];
#pragma unroll
        for (int n = 0; n < NT8; n++) {
            const float e0 = ex2(s[n][0] - m_use[0]), e1 = ex2(s[n][1] - m_use[0]);
            const float e2 = ex2(s[n][2] - m_use[1]), e3 = ex2(s[n][3] - m_use[1]);
            rs[0] += e0 + e1, rs[1] += e2 + e3;
            pa[n >> 1][(n & 1) * 2] = pack_bf16(e0, e1);
            pa[n >> 1][(n & 1) * 2 + 1] = pack_bf16(e2, e3);
        }
#pragma unroll
        for (int h = 0; h < 2; h++) l_run[h] = fmaf(l_run[h], alpha[h], rs[h]);  // per lane; the quad's lanes meet at the end
        if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
            for (int n = 0; n < NO; n++) o[n][0] *= alpha[0], o[n][1] *= alpha[0], o[n][2] *= alpha[1], o[n][3] *= alpha[1];
        }
#pragma unroll
        for (int kk = 0; kk < KK; kk++) {
#pragma unroll
            for (int np = 0; np < NO / 2; np++) {
                uint32_t b[4];
                ldsm4_t(b, vt + G::off(tok0 + kk * 16 + (lane & 15), np * 2 + (lane >> 4)));
                mma_bf16(o[2 * np], pa[kk], b[0], b[1]);
                mma_bf16(o[2 * np + 1], pa[kk], b[2], b[3]);
            }
        }
        __syncthreads();  // a stage is rewritten only after every warp is done with it
        if (tile + NST < n_tiles) issue(tile + NST, stage);
        else cp_async_commit();
    }
    cp_async_wait<0>();
    pdl_launch_dependents();
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
    }

    const int64_t tile_id = (int64_t)blockIdx.z * a.keys.kv_heads + kvh;
    const int64_t share = (tile_id * n_splits + blockIdx.x) * QT;
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out);
    auto out_at = [&](int qi) { return out + (int64_t)(row_first + qi / grp) * a.out_stride + (kvh * grp + qi % grp) * D; };

    if (SL == 1) {
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int qi = mt * 16 + gid + 8 * h;
            if (qi >= n_queries) continue;
            if (n_splits == 1) {
                const int row = row_first + qi / grp, head = kvh * grp + qi % grp;
                const float f = head_factor(a, row, head, m_run[h], l_run[h]);
                __nv_bfloat16* p = out_at(qi);
#pragma unroll
                for (int n = 0; n < NO; n++) {
                    float2 v = make_float2(o[n][2 * h] * f, o[n][2 * h + 1] * f);
                    if (a.turn) turn_back(a, row, n * 8 + 2 * tig, v.x, v.y);
                    if (a.value_gate) v.x *= value_gate(a, row, head, n * 8 + 2 * tig), v.y *= value_gate(a, row, head, n * 8 + 2 * tig + 1);
                    *reinterpret_cast<uint32_t*>(p + n * 8 + 2 * tig) = pack_bf16(v.x, v.y);
                }
            } else {
                float* p = part_o + (share + qi) * D;
#pragma unroll
                for (int n = 0; n < NO; n++) *reinterpret_cast<float2*>(p + n * 8 + 2 * tig) = make_float2(o[n][2 * h], o[n][2 * h + 1]);
                if (tig == 0) part_ml[share + qi] = make_float2(m_run[h], l_run[h]);
            }
        }
    } else {
        // the slices of an m-tile meet in shared memory (the ring is free now)
        constexpr int DP = D + 4;
        float* wo = reinterpret_cast<float*>(smem);
        float2* wml = reinterpret_cast<float2*>(smem + (size_t)MT * SL * 16 * DP * 4);
        __syncthreads();
        float* dst = wo + (size_t)warp * 16 * DP;
#pragma unroll
        for (int n = 0; n < NO; n++) {
            *reinterpret_cast<float2*>(dst + gid * DP + n * 8 + 2 * tig) = make_float2(o[n][0], o[n][1]);
            *reinterpret_cast<float2*>(dst + (gid + 8) * DP + n * 8 + 2 * tig) = make_float2(o[n][2], o[n][3]);
        }
        if (tig == 0) {
            wml[warp * 16 + gid] = make_float2(m_run[0], l_run[0]);
            wml[warp * 16 + gid + 8] = make_float2(m_run[1], l_run[1]);
        }
        __syncthreads();
        finish_slices<D, QT, SL, NTHR, false>(a, row_first, kvh, grp, n_queries, n_splits, wo, wml, part_o, part_ml, tickets);
    }
}

// ------------------------------------------------------------------ up to 32 queries per key head
// The queries of a decoded token or a verify pass fill the N side of the mma in tiles of eight, the keys its M side:
// S^T = K Q^T and O^T = K^T P^T.  Hardly a multiply or an exponential goes to empty query slots, a key fragment serves every
// query tile, and one query tile needs so few registers that four CTAs share an SM.  Four warps, each a quarter of every
// key tile.
template <int D, int NQ, bool KV>
struct FewQ {
    static constexpr int TILE = D <= 64 ? 128 : 64;   // tokens per key tile: 16 KB and more in flight per stage
    static constexpr int NST = ring_stages<D, KV>(), V_AT = KV ? TILE * Geo<D>::PITCH : 0, STAGE = TILE * Geo<D>::PITCH + V_AT;
    static constexpr int WTOK = TILE / 4, NK = WTOK / 16;
    static constexpr size_t RING = (size_t)NST * STAGE;
    static constexpr size_t MERGE = (size_t)4 * 8 * NQ * ((D + 4) * 4 + 8);
    static constexpr size_t SMEM = RING > MERGE ? RING : MERGE;
    static constexpr int PER_SM = D > 128 ? 2 : NQ == 1 ? 4 : NQ == 2 ? 3 : 2;
};

template <int D, int NQ, bool KV, bool PRE>
__global__ void __launch_bounds__(128, FewQ<D, NQ, KV>::PER_SM)
    window_attn_few_kernel(const __grid_constant__ WindowAttn a, const AttnTile* __restrict__ tiles, int rows_per_seq, float* __restrict__ part_o,
                        float2* __restrict__ part_ml, uint32_t* __restrict__ tickets, uint32_t* __restrict__ err) {
    using G = Geo<D>;
    using F = FewQ<D, NQ, KV>;
    constexpr int KS = D / 16, NM = D / 16, NK = F::NK, QT = 8 * NQ, NST = F::NST;
    extern __shared__ __align__(128) uint8_t smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int kvh = blockIdx.y, n_splits = gridDim.x;
    const int grp = a.n_q_heads / a.keys.kv_heads;
    const int row_first = tiles ? tiles[blockIdx.z].row_first : (int)blockIdx.z * rows_per_seq;
    const int n_rows = tiles ? tiles[blockIdx.z].n_rows : rows_per_seq;
    const tsb_row_desc rd0 = a.rows[row_first];
    const int seq = rd0.seq, pos0 = rd0.base + rd0.slot;
    const int n_queries = n_rows * grp;
    if (seq < 0 || seq >= a.keys.max_seqs || n_queries > QT) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        pdl_wait();
        return;
    }
    // key tiles start at multiples of 64 positions; this CTA's run of them
    const int lo = first_visible(a, pos0) & ~63;
    const int hi = pos0 + n_rows, lo_last = first_visible(a, hi - 1);
    const int n_pre = PRE ? prefix_len(a, hi - 1) : 0, pre_all = PRE ? prefix_len(a, pos0) : 0;  // of the prefix: seen by some row, by every row
    const int pre_tiles = (n_pre + F::TILE - 1) / F::TILE;
    const int total = pre_tiles + (hi - lo + F::TILE - 1) / F::TILE;
    const int per = (total + n_splits - 1) / n_splits;
    const int t_first = min(total, (int)blockIdx.x * per), n_tiles = min(total, t_first + per) - t_first;
    const int begin = lo + (t_first - pre_tiles) * F::TILE;

    const uint32_t ring = smem_u32(smem);
    auto issue = [&](int tile, int stage) {
        constexpr int TPR = 128 / F::TILE;  // threads per token row
        const int r = threadIdx.x / TPR, part = threadIdx.x % TPR;
        const bool pre = PRE && t_first + tile < pre_tiles;
        const int pos = (pre ? (t_first + tile) * F::TILE : begin + tile * F::TILE) + r;
        const __nv_bfloat16* src = pos >= (pre ? n_pre : hi) ? nullptr : PRE ? run_row(a, pre, seq, pos) : key_row<__nv_bfloat16>(a.keys, seq, pos);
        const bool ok = src != nullptr;
        src = ok ? src + (int64_t)kvh * a.keys.head_step : reinterpret_cast<const __nv_bfloat16*>(a.keys.base);
        const uint32_t dst = ring + stage * F::STAGE;
#pragma unroll
        for (int c = part; c < G::CH; c += TPR) cp16(dst + G::off(r, c), ok ? src + c * 8 : src, ok);
        if (KV) {
#pragma unroll
            for (int c = part; c < G::CH; c += TPR) cp16(dst + F::V_AT + G::off(r, c), ok ? src + a.keys.value_off + c * 8 : src, ok);
        }
        cp_async_commit();
    };
    auto prologue = [&]() {
#pragma unroll
        for (int i = 0; i < NST; i++) {
            if (i < n_tiles) issue(i, i);
            else cp_async_commit();
        }
    };
    // key tiles of earlier passes, prefix rows of their positions
    const bool early = begin + NST * F::TILE <= rd0.base && (!PRE || min(n_pre, (t_first + NST) * F::TILE) * max(a.pool, 1) <= rd0.base);
    if (early) prologue();
    // score columns of this lane: queries 2 tig and 2 tig + 1 of every query tile
    int pq[NQ][2];
    float r1[NQ][2], r2[NQ][2], span[NQ][2];
#pragma unroll
    for (int q = 0; q < NQ; q++)
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int qi = q * 8 + 2 * tig + h;
            const bool v = qi < n_queries;
            const int head = kvh * grp + (v ? qi % grp : 0);
            pq[q][h] = pos0 + (v ? qi / grp : 0);  // an empty slot repeats the first query and is not stored
            r1[q][h] = a.slopes ? a.slopes[head] * 1.4426950408889634f : a.r1 ? a.r1[head] : 0.f, r2[q][h] = a.r1 ? a.r2[head] : 0.f;
            span[q][h] = visible_span(a, pq[q][h]);
        }
    pdl_wait();
    if (!early) prologue();
    // Q^T fragments: lane column n = query gid of the tile
    uint32_t qb[NQ][KS][2];
#pragma unroll
    for (int q = 0; q < NQ; q++) {
        const int qi = q * 8 + gid;
        const bool v = qi < n_queries;
        const uint32_t* p = reinterpret_cast<const uint32_t*>(reinterpret_cast<const __nv_bfloat16*>(a.q) + (int64_t)(row_first + (v ? qi / grp : 0)) * a.q_stride +
                                                              (kvh * grp + (v ? qi % grp : 0)) * D);
#pragma unroll
        for (int ks = 0; ks < KS; ks++) qb[q][ks][0] = p[8 * ks + tig], qb[q][ks][1] = p[8 * ks + 4 + tig];
    }
    const ScoreConst sc(a);
    float o[NQ][NM][4];
    float m_run[NQ][2], l_run[NQ][2];
#pragma unroll
    for (int q = 0; q < NQ; q++) {
#pragma unroll
        for (int n = 0; n < NM; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) o[q][n][i] = 0.f;
        m_run[q][0] = m_run[q][1] = -INFINITY, l_run[q][0] = l_run[q][1] = 0.f;
    }
    for (int tile = 0; tile < n_tiles; tile++) {
        const int stage = tile % NST;
        cp_async_wait<NST - 1>();
        __syncthreads();
        const uint32_t kt = ring + stage * F::STAGE, vt = kt + F::V_AT;
        const bool pre = PRE && t_first + tile < pre_tiles;
        const int tok0 = warp * F::WTOK, p0 = (pre ? (t_first + tile) * F::TILE : begin + tile * F::TILE) + tok0;
        float s[NQ][NK][4];  // rows gid, gid + 8 of sixteen keys x the lane's two queries
#pragma unroll
        for (int n = 0; n < NK; n++) {
#pragma unroll
            for (int q = 0; q < NQ; q++)
#pragma unroll
                for (int i = 0; i < 4; i++) s[q][n][i] = 0.f;
#pragma unroll
            for (int ks = 0; ks < KS; ks++) {
                uint32_t k[4];
                ldsm4(k, kt + G::off(tok0 + n * 16 + (lane & 15), ks * 2 + (lane >> 4)));
#pragma unroll
                for (int q = 0; q < NQ; q++) mma_bf16(s[q][n], k, qb[q][ks][0], qb[q][ks][1]);
            }
        }
        const bool edge = pre ? p0 + F::WTOK > pre_all : p0 + F::WTOK > pos0 || p0 < lo_last;
        uint32_t pb[NQ][NK][2];
#pragma unroll
        for (int q = 0; q < NQ; q++) {
            float mx[2] = {-INFINITY, -INFINITY}, db[2], sp[2];
#pragma unroll
            for (int h = 0; h < 2; h++) {
                const int last = pre ? prefix_len(a, pq[q][h]) - 1 : pq[q][h];
                db[h] = (float)(last - p0 - gid), sp[h] = pre ? 3e38f : span[q][h];
            }
            base2_logits<NK, true>(s[q], a, sc, db, r1[q], r2[q], sp, edge, mx);
            float alpha[2], m_use[2];
#pragma unroll
            for (int h = 0; h < 2; h++) {
#pragma unroll
                for (int o2 = 4; o2 < 32; o2 <<= 1) mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], o2));
                const float m_new = fmaxf(m_run[q][h], mx[h]);
                m_use[h] = m_new == -INFINITY ? 0.f : m_new;
                alpha[h] = ex2(m_run[q][h] - m_use[h]);
                m_run[q][h] = m_new;
                l_run[q][h] *= alpha[h];
            }
            if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
                for (int n = 0; n < NM; n++) o[q][n][0] *= alpha[0], o[q][n][1] *= alpha[1], o[q][n][2] *= alpha[0], o[q][n][3] *= alpha[1];
            }
#pragma unroll
            for (int n = 0; n < NK; n++) {
                const float e0 = ex2(s[q][n][0] - m_use[0]), e1 = ex2(s[q][n][1] - m_use[1]), e2 = ex2(s[q][n][2] - m_use[0]), e3 = ex2(s[q][n][3] - m_use[1]);
                l_run[q][0] += e0 + e2, l_run[q][1] += e1 + e3;
                // (keys x queries) fragments to the B operand's (keys along the registers): an 8 x 8 transpose each
                uint32_t b0 = pack_bf16(e0, e1), b1 = pack_bf16(e2, e3);
                asm("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(pb[q][n][0]) : "r"(b0));
                asm("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(pb[q][n][1]) : "r"(b1));
            }
        }
#pragma unroll
        for (int n = 0; n < NK; n++)
#pragma unroll
            for (int m = 0; m < NM; m++) {
                // V^T: rows = columns of the head, from the value rows through the transposing load
                uint32_t k[4];
                ldsm4_t(k, vt + G::off(tok0 + n * 16 + ((lane >> 4) << 3) + (lane & 7), m * 2 + ((lane >> 3) & 1)));
#pragma unroll
                for (int q = 0; q < NQ; q++) mma_bf16(o[q][m], k, pb[q][n][0], pb[q][n][1]);
            }
        __syncthreads();  // a stage is rewritten only after every warp is done with it
        if (tile + NST < n_tiles) issue(tile + NST, stage);
        else cp_async_commit();
    }
    cp_async_wait<0>();
    pdl_launch_dependents();
    constexpr int DP = D + 4;
    float* wo = reinterpret_cast<float*>(smem);
    float2* wml = reinterpret_cast<float2*>(smem + (size_t)4 * QT * DP * 4);
    __syncthreads();
#pragma unroll
    for (int q = 0; q < NQ; q++) {
#pragma unroll
        for (int h = 0; h < 2; h++)
#pragma unroll
            for (int o2 = 4; o2 < 32; o2 <<= 1) l_run[q][h] += __shfl_xor_sync(0xffffffffu, l_run[q][h], o2);
        const int slot = warp * QT + q * 8 + 2 * tig;
#pragma unroll
        for (int m = 0; m < NM; m++)
#pragma unroll
            for (int i = 0; i < 4; i++) wo[(size_t)(slot + (i & 1)) * DP + m * 16 + gid + (i >> 1) * 8] = o[q][m][i];
        if (gid == 0) wml[slot] = make_float2(m_run[q][0], l_run[q][0]), wml[slot + 1] = make_float2(m_run[q][1], l_run[q][1]);
    }
    __syncthreads();
    finish_slices<D, QT, 4, 128, NQ == 1>(a, row_first, kvh, grp, n_queries, n_splits, wo, wml, part_o, part_ml, tickets);
}

template <int D, int MT, int SL, bool KV, bool PRE = false>
cudaError_t launch_one(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    const int splits = wattn_splits(ctx, a, l, TOK, 16 * MT, SL == 1 ? 1 : MT == 1 ? 3 : 2);
    const WattnScratch sc = wattn_scratch(ctx, scratch);
    constexpr size_t smem = wattn_smem<D, MT, SL, KV>();
    static SmemOptIn configured;
    if (cudaError_t e = tsb_opt_in_smem(ctx, window_attn_kernel<D, MT, SL, KV, PRE>, smem, configured); e != cudaSuccess) return e;
    cudaError_t e = tsb_launch(ctx, window_attn_kernel<D, MT, SL, KV, PRE>, dim3((unsigned)splits, (unsigned)a.keys.kv_heads, (unsigned)l.n_tiles), dim3(32 * MT * SL),
                               smem, st, true, a, l.tiles, l.tiles_per_group, l.rows_per_seq, l.rows_per_tile, sc.o, sc.ml, sc.tickets, ctx->dev_error);
    return e == cudaSuccess && splits > 1 ? launch_window_attn_merge(ctx, st, a, l, splits, 16 * MT, sc) : e;
}

template <int D, int NQ, bool KV, bool PRE>
cudaError_t launch_few(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    using F = FewQ<D, NQ, KV>;
    const int splits = wattn_splits(ctx, a, l, F::TILE, 8 * NQ, F::PER_SM);
    const WattnScratch sc = wattn_scratch(ctx, scratch);
    static SmemOptIn configured;
    if (cudaError_t e = tsb_opt_in_smem(ctx, window_attn_few_kernel<D, NQ, KV, PRE>, F::SMEM, configured); e != cudaSuccess) return e;
    cudaError_t e = tsb_launch(ctx, window_attn_few_kernel<D, NQ, KV, PRE>, dim3((unsigned)splits, (unsigned)a.keys.kv_heads, (unsigned)l.n_tiles), dim3(128), F::SMEM,
                               st, true, a, l.tiles, l.rows_per_seq, sc.o, sc.ml, sc.tickets, ctx->dev_error);
    return e == cudaSuccess && splits > 1 && NQ > 1 ? launch_window_attn_merge(ctx, st, a, l, splits, 8 * NQ, sc) : e;
}
// query tiles by the number of queries; head sizes above 128 have registers for one
template <int D, bool KV, bool PRE>
cudaError_t launch_few_dim(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int queries, void* scratch) {
    if (queries <= 8) return launch_few<D, 1, KV, PRE>(ctx, st, a, l, scratch);
    if (queries <= 16) return launch_one<D, 1, 4, KV, PRE>(ctx, st, a, l, scratch);  // sixteen query rows of one mma tile: faster than two tiles of eight
    if constexpr (D <= 128) {
        if (queries <= 24) return launch_few<D, 3, KV, PRE>(ctx, st, a, l, scratch);
        if (queries <= 32) return launch_few<D, 4, KV, PRE>(ctx, st, a, l, scratch);
    }
    return launch_one<D, 4, 2, KV, PRE>(ctx, st, a, l, scratch);
}

template <int MT, int SL, bool KV, bool PRE = false>
cudaError_t launch_large(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    switch (a.keys.head_dim) {
        case 32: return launch_one<32, MT, SL, KV, PRE>(ctx, st, a, l, scratch);
        case 64: return launch_one<64, MT, SL, KV, PRE>(ctx, st, a, l, scratch);
        case 96: return launch_one<96, MT, SL, KV, PRE>(ctx, st, a, l, scratch);
        case 128: return launch_one<128, MT, SL, KV, PRE>(ctx, st, a, l, scratch);
        case 192: return launch_one<192, MT, SL, KV, PRE>(ctx, st, a, l, scratch);
        case 256: return launch_one<256, MT, SL, KV, PRE>(ctx, st, a, l, scratch);
        default: return cudaErrorInvalidValue;
    }
}

template <bool KV, bool PRE = false>
cudaError_t launch_small(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int queries, void* scratch) {
    switch (a.keys.head_dim) {
        case 32: return launch_few_dim<32, KV, PRE>(ctx, st, a, l, queries, scratch);
        case 64: return launch_few_dim<64, KV, PRE>(ctx, st, a, l, queries, scratch);
        case 96: return launch_few_dim<96, KV, PRE>(ctx, st, a, l, queries, scratch);
        case 128: return launch_few_dim<128, KV, PRE>(ctx, st, a, l, queries, scratch);
        case 192: return launch_few_dim<192, KV, PRE>(ctx, st, a, l, queries, scratch);
        case 256: return launch_few_dim<256, KV, PRE>(ctx, st, a, l, queries, scratch);
        default: return cudaErrorInvalidValue;
    }
}


}  // namespace
