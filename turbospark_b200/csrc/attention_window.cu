// Sliding-window attention over a key-only paged cache (attention_window.cuh).
//
// bfloat16: one kernel template <D, MT, SL> on mma.sync m16n8k16.  A CTA owns one (query tile, key head, run of key tiles):
// MT m-tiles of 16 queries - the tile's rows x the heads that share the key head - and walks 64-token key tiles that
// cp.async brings into a three-stage ring.  The one tile in shared memory serves both products: K rows as the B operand
// of S = Q K^T (ldmatrix) and as the B operand of O += P K (ldmatrix.trans), so a key byte is read once.  SL warps share an
// m-tile, each taking 64 / SL tokens of every tile, and meet at the end.
//   few queries (short portions): MT = 1 or 4, SL = 4 or 2; many queries whose geometry the tcgen05 kernel (attention_window_tc.cu) does
//   not take: MT = 8, SL = 1
// Up to eight queries per key head (decoded tokens), and 17 to 32 (verify passes) with heads of up to 128 columns, go to
// window_attn_few_kernel: keys on the M side.
// A context that does not fill the device with CTAs is cut into runs of key tiles: with up to eight queries the last CTA of a
// tile to finish - decided by a ticket, nobody waits - adds the runs in order, with more a merge launch does.
// Only the key tiles inside the window of some query of the tile are visited; key tiles start at multiples of 64 positions
// whatever the cut of the prompt, so a row meets its keys in the same grouping in every schedule.
//
// Score arithmetic in f32, base 2: v = cap log2(e) tanh(s scale / cap) - r1 log2(1 + r2 d); tanh by its series where every
// score of the warp's tile is well inside the cap.
//
// f32: one warp per (row, query head), lanes over keys for the scores and over columns for the sum; the reference-precision
// mode, plain fused multiply-adds and the library's exp, tanh and log.
#include <algorithm>

#include "attention_window_dev.cuh"

namespace {

constexpr int TOK = 64;   // tokens per key tile
constexpr int NST = 3;    // key tiles in flight

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
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
// db[h]: distance of the lane's first key from its query h.
template <int N, bool KEYS_M>
__device__ __forceinline__ void base2_logits(float (&s)[N][4], const WindowAttn& a, const ScoreConst& sc, const float (&db)[2], const float (&r1)[2],
                                             const float (&r2)[2], bool edge, float (&mx)[2]) {
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
                    const float2 x = make_float2(s[n][i], s[n][i + 1]), z = mul2(x, x);
                    const float2 v = mul2(x, fma2(z, fma2(z, fma2(z, fma2(z, both(sc.k4), both(sc.k3)), both(sc.k2)), both(sc.k1)), both(sc.k0)));
                    s[n][i] = v.x, s[n][i + 1] = v.y;
                }
        }
    } else {
#pragma unroll
        for (int n = 0; n < N; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) s[n][i] *= sc.s_in;
    }
    const float window = a.window > 0 ? (float)a.window : 3e38f;
#pragma unroll
    for (int n = 0; n < N; n++)
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int h = KEYS_M ? i & 1 : i >> 1;
            const float dist = db[h] - (float)(KEYS_M ? n * 16 + (i >> 1) * 8 : n * 8 + (i & 1));
            if (a.r1) s[n][i] = fmaf(-r1[h], lg2(fmaf(r2[h], dist, 1.f)), s[n][i]);
            if (edge && (dist < 0.f || dist >= window)) s[n][i] = -INFINITY;
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
    auto store = [&](int qi, int c, float4 v, float l) {  // 1 / sum, times the head's gate
        const int row = row_first + qi / grp, head = kvh * grp + qi % grp;
        float f = l > 0.f ? 1.f / l : 0.f;
        if (a.gate) f *= sigmoid(a.gate[(int64_t)row * a.n_q_heads + head]);
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
            store(qi, c, acc, l);
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
        store(qi, c, acc, l);
    }
}

template <int D, int MT, int SL>
constexpr size_t wattn_smem() {
    const size_t ring = (size_t)NST * TOK * Geo<D>::PITCH + (SL == 1 ? (size_t)MT * 16 * Geo<D>::PITCH : 0);
    const size_t merge = SL > 1 ? (size_t)MT * SL * 16 * ((D + 4) * 4 + 8) : 0;
    return ring > merge ? ring : merge;
}

template <int D, int MT, int SL>
__global__ void __launch_bounds__(32 * MT * SL, MT * SL <= 4 ? 3 : 1)
    window_attn_kernel(const __grid_constant__ WindowAttn a, const AttnTile* __restrict__ tiles, int tiles_per_group, int rows_per_seq, int rows_per_tile,
                       float* __restrict__ part_o, float2* __restrict__ part_ml, uint32_t* __restrict__ tickets, uint32_t* __restrict__ err) {
    using G = Geo<D>;
    constexpr int KS = D / 16, NO = D / 8, QT = 16 * MT, NTHR = 32 * MT * SL;
    constexpr int WTOK = TOK / SL, NT8 = WTOK / 8, KK = WTOK / 16;
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
    const int lo = a.window > 0 ? max(0, pos0 - a.window + 1) & ~(TOK - 1) : 0;
    const int hi = pos0 + n_rows;
    const int total = (hi - lo + TOK - 1) / TOK;
    const int per = (total + n_splits - 1) / n_splits;
    const int t_first = min(total, (int)blockIdx.x * per), n_tiles = min(total, t_first + per) - t_first;
    const int begin = lo + t_first * TOK;

    const uint32_t ring = smem_u32(smem);
    auto issue = [&](int tile, int stage) {
        constexpr int TPR = NTHR / TOK;  // threads per token row
        const int r = threadIdx.x / TPR, part = threadIdx.x % TPR;
        const int pos = begin + tile * TOK + r;
        const __nv_bfloat16* src = pos < hi ? key_row<__nv_bfloat16>(a.keys, seq, pos) : nullptr;
        const bool ok = src != nullptr;
        src = ok ? src + (int64_t)kvh * D : reinterpret_cast<const __nv_bfloat16*>(a.keys.base);
        const uint32_t dst = ring + stage * (TOK * G::PITCH);
#pragma unroll
        for (int c = part; c < G::CH; c += TPR) cp16(dst + G::off(r, c), ok ? src + c * 8 : src, ok);
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
    const bool early = begin + NST * TOK <= rd0.base;
    if (early) prologue();
    pdl_wait();
    if (!early) prologue();

    // the lane's two queries: rows gid and gid + 8 of its m-tile
    const __nv_bfloat16* qp[2];
    int pq[2];
    float r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int qi = mt * 16 + gid + 8 * h;
        const bool v = qi < n_queries;
        const int row = v ? qi / grp : 0, head = kvh * grp + (v ? qi % grp : 0);
        pq[h] = pos0 + row;  // an empty slot repeats the first query and is not stored
        qp[h] = reinterpret_cast<const __nv_bfloat16*>(a.q) + (int64_t)(row_first + row) * a.q_stride + head * D;
        if (a.r1) r1[h] = a.r1[head], r2[h] = a.r2[head];
    }
    uint32_t qa[QREG ? KS : 1][4];
    const uint32_t q_smem = ring + NST * TOK * G::PITCH;
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
            *reinterpret_cast<uint4*>(smem + NST * TOK * G::PITCH + G::off(qi, c)) = v;
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
        const uint32_t kt = ring + stage * (TOK * G::PITCH);
        const int tok0 = sl * WTOK;
        const int p0 = begin + tile * TOK + tok0;
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
        const bool edge = p0 + WTOK > pos0 || (a.window > 0 && p0 <= pos0 + n_rows - 1 - a.window);
        float mx[2] = {-INFINITY, -INFINITY};
        const float db[2] = {(float)(pq[0] - p0 - 2 * tig), (float)(pq[1] - p0 - 2 * tig)};
        base2_logits<NT8, false>(s, a, sc, db, r1, r2, edge, mx);
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
                ldsm4_t(b, kt + G::off(tok0 + kk * 16 + (lane & 15), np * 2 + (lane >> 4)));
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
    auto factor = [&](int qi, float l) {  // 1 / sum, times the head's gate
        const float inv = l > 0.f ? 1.f / l : 0.f;
        return a.gate ? inv * sigmoid(a.gate[(int64_t)(row_first + qi / grp) * a.n_q_heads + kvh * grp + qi % grp]) : inv;
    };

    if (SL == 1) {
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int qi = mt * 16 + gid + 8 * h;
            if (qi >= n_queries) continue;
            if (n_splits == 1) {
                const float f = factor(qi, l_run[h]);
                __nv_bfloat16* p = out_at(qi);
#pragma unroll
                for (int n = 0; n < NO; n++) *reinterpret_cast<uint32_t*>(p + n * 8 + 2 * tig) = pack_bf16(o[n][2 * h] * f, o[n][2 * h + 1] * f);
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
template <int D, int NQ>
struct FewQ {
    static constexpr int TILE = D <= 64 ? 128 : 64;   // tokens per key tile: 16 KB and more in flight per stage
    static constexpr int WTOK = TILE / 4, NK = WTOK / 16;
    static constexpr size_t RING = (size_t)NST * TILE * Geo<D>::PITCH;
    static constexpr size_t MERGE = (size_t)4 * 8 * NQ * ((D + 4) * 4 + 8);
    static constexpr size_t SMEM = RING > MERGE ? RING : MERGE;
    static constexpr int PER_SM = D > 128 ? 2 : NQ == 1 ? 4 : NQ == 2 ? 3 : 2;
};

template <int D, int NQ>
__global__ void __launch_bounds__(128, FewQ<D, NQ>::PER_SM)
    window_attn_few_kernel(const __grid_constant__ WindowAttn a, const AttnTile* __restrict__ tiles, int rows_per_seq, float* __restrict__ part_o,
                        float2* __restrict__ part_ml, uint32_t* __restrict__ tickets, uint32_t* __restrict__ err) {
    using G = Geo<D>;
    using F = FewQ<D, NQ>;
    constexpr int KS = D / 16, NM = D / 16, NK = F::NK, QT = 8 * NQ;
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
    const int lo = a.window > 0 ? max(0, pos0 - a.window + 1) & ~63 : 0;
    const int hi = pos0 + n_rows;
    const int total = (hi - lo + F::TILE - 1) / F::TILE;
    const int per = (total + n_splits - 1) / n_splits;
    const int t_first = min(total, (int)blockIdx.x * per), n_tiles = min(total, t_first + per) - t_first;
    const int begin = lo + t_first * F::TILE;

    const uint32_t ring = smem_u32(smem);
    auto issue = [&](int tile, int stage) {
        constexpr int TPR = 128 / F::TILE;  // threads per token row
        const int r = threadIdx.x / TPR, part = threadIdx.x % TPR;
        const int pos = begin + tile * F::TILE + r;
        const __nv_bfloat16* src = pos < hi ? key_row<__nv_bfloat16>(a.keys, seq, pos) : nullptr;
        const bool ok = src != nullptr;
        src = ok ? src + (int64_t)kvh * D : reinterpret_cast<const __nv_bfloat16*>(a.keys.base);
        const uint32_t dst = ring + stage * (F::TILE * G::PITCH);
#pragma unroll
        for (int c = part; c < G::CH; c += TPR) cp16(dst + G::off(r, c), ok ? src + c * 8 : src, ok);
        cp_async_commit();
    };
    auto prologue = [&]() {
#pragma unroll
        for (int i = 0; i < NST; i++) {
            if (i < n_tiles) issue(i, i);
            else cp_async_commit();
        }
    };
    const bool early = begin + NST * F::TILE <= rd0.base;  // key tiles of earlier passes
    if (early) prologue();
    // score columns of this lane: queries 2 tig and 2 tig + 1 of every query tile
    int pq[NQ][2];
    float r1[NQ][2], r2[NQ][2];
#pragma unroll
    for (int q = 0; q < NQ; q++)
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int qi = q * 8 + 2 * tig + h;
            const bool v = qi < n_queries;
            const int head = kvh * grp + (v ? qi % grp : 0);
            pq[q][h] = pos0 + (v ? qi / grp : 0);  // an empty slot repeats the first query and is not stored
            r1[q][h] = a.r1 ? a.r1[head] : 0.f, r2[q][h] = a.r1 ? a.r2[head] : 0.f;
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
        const uint32_t kt = ring + stage * (F::TILE * G::PITCH);
        const int tok0 = warp * F::WTOK, p0 = begin + tile * F::TILE + tok0;
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
        const bool edge = p0 + F::WTOK > pos0 || (a.window > 0 && p0 <= pos0 + n_rows - 1 - a.window);
        uint32_t pb[NQ][NK][2];
#pragma unroll
        for (int q = 0; q < NQ; q++) {
            float mx[2] = {-INFINITY, -INFINITY};
            const float db[2] = {(float)(pq[q][0] - p0 - gid), (float)(pq[q][1] - p0 - gid)};
            base2_logits<NK, true>(s[q], a, sc, db, r1[q], r2[q], edge, mx);
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
                // K^T: rows = columns of the head, from the key rows through the transposing load
                uint32_t k[4];
                ldsm4_t(k, kt + G::off(tok0 + n * 16 + ((lane >> 4) << 3) + (lane & 7), m * 2 + ((lane >> 3) & 1)));
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

// ------------------------------------------------------------------ merge of cut tiles
// One CTA per row and eight query heads, a warp per head: the runs' weights sit in the lanes, the sums go over the runs in order.
__global__ void __launch_bounds__(256)
    window_attn_merge_kernel(const __grid_constant__ WindowAttn a, const AttnTile* __restrict__ tiles, int tiles_per_group, int rows_per_seq,
                             int rows_per_tile, int n_splits, int slots, const float* __restrict__ part_o, const float2* __restrict__ part_ml) {
    const int tile = blockIdx.x, r = blockIdx.y;
    int row_first, n_rows;
    if (tiles) {
        row_first = tiles[tile].row_first, n_rows = tiles[tile].n_rows;
    } else {
        const int in_group = (tile % tiles_per_group) * rows_per_tile;
        row_first = (tile / tiles_per_group) * rows_per_seq + in_group;
        n_rows = min(rows_per_tile, rows_per_seq - in_group);
    }
    pdl_wait();
    pdl_launch_dependents();
    if (r >= n_rows) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int D = a.keys.head_dim, grp = a.n_q_heads / a.keys.kv_heads, R = WATTN_LARGE_Q / grp;
    const int head = blockIdx.z * 8 + warp;
    if (head < a.n_q_heads) {
        const int slot = (r / R) * WATTN_LARGE_Q + (r % R) * grp + head % grp;
        const int64_t first = ((int64_t)tile * a.keys.kv_heads + head / grp) * n_splits * slots + slot;
        float2 v[WATTN_MAX_SPLITS / 32];
        float m = -INFINITY, l = 0.f;
#pragma unroll
        for (int i = 0; i < WATTN_MAX_SPLITS / 32; i++) {
            const int k = i * 32 + lane;
            v[i] = k < n_splits ? part_ml[first + (int64_t)k * slots] : make_float2(-INFINITY, 0.f);
            m = fmaxf(m, v[i].x);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        const float mu = m == -INFINITY ? 0.f : m;
#pragma unroll
        for (int i = 0; i < WATTN_MAX_SPLITS / 32; i++) v[i].x = ex2(v[i].x - mu), l = fmaf(v[i].y, v[i].x, l);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
        float f = l > 0.f ? 1.f / l : 0.f;
        if (a.gate) f *= sigmoid(a.gate[(int64_t)(row_first + r) * a.n_q_heads + head]);
        __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (int64_t)(row_first + r) * a.out_stride + (int64_t)head * D;
        for (int c0 = 0; c0 < D; c0 += 128) {
            const int c = c0 + lane * 4;
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
            for (int k = 0; k < n_splits; k++) {
                const float w = __shfl_sync(0xffffffffu, k < 32 ? v[0].x : v[1].x, k & 31);
                if (c < D) {
                    const float4 x = *reinterpret_cast<const float4*>(part_o + (first + (int64_t)k * slots) * D + c);
                    acc.x = fmaf(x.x, w, acc.x), acc.y = fmaf(x.y, w, acc.y), acc.z = fmaf(x.z, w, acc.z), acc.w = fmaf(x.w, w, acc.w);
                }
            }
            if (c < D) *reinterpret_cast<uint2*>(out + c) = make_uint2(pack_bf16(acc.x * f, acc.y * f), pack_bf16(acc.z * f, acc.w * f));
        }
    }
}

// ------------------------------------------------------------------ f32
constexpr int F32_WARPS = 4;
constexpr int F32_MAX_DIM = 512;
__global__ void __launch_bounds__(F32_WARPS * 32) window_attn_f32_kernel(const __grid_constant__ WindowAttn a, int rows, uint32_t* __restrict__ err) {
    __shared__ float qs[F32_WARPS][F32_MAX_DIM];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t item = (int64_t)blockIdx.x * F32_WARPS + warp;
    pdl_wait();
    pdl_launch_dependents();
    if (item >= (int64_t)rows * a.n_q_heads) return;
    const int row = (int)(item / a.n_q_heads), head = (int)(item % a.n_q_heads);
    const int D = a.keys.head_dim, kvh = head / (a.n_q_heads / a.keys.kv_heads);
    const tsb_row_desc rd = a.rows[row];
    const int pos = rd.base + rd.slot;
    const float* q = reinterpret_cast<const float*>(a.q) + (int64_t)row * a.q_stride + (int64_t)head * D;
    for (int i = lane; i < D; i += 32) qs[warp][i] = q[i];
    __syncwarp();
    const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    const float r1 = a.r1 ? a.r1[head] : 0.f, r2 = a.r1 ? a.r2[head] : 0.f;
    float m = -INFINITY, l = 0.f, acc[F32_MAX_DIM / 32];
#pragma unroll
    for (int i = 0; i < F32_MAX_DIM / 32; i++) acc[i] = 0.f;
    for (int j0 = lo & ~31; j0 <= pos; j0 += 32) {
        const int j = j0 + lane;
        const bool seen = j >= lo && j <= pos;
        const float* k = seen ? key_row<float>(a.keys, rd.seq, j) : nullptr;
        if (seen && !k) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        float s = -INFINITY;
        if (k) {
            k += (int64_t)kvh * D;
            float dot = 0.f;
            for (int i = 0; i < D; i += 4) {
                const float4 v = *reinterpret_cast<const float4*>(k + i);
                dot = fmaf(v.x, qs[warp][i], dot), dot = fmaf(v.y, qs[warp][i + 1], dot);
                dot = fmaf(v.z, qs[warp][i + 2], dot), dot = fmaf(v.w, qs[warp][i + 3], dot);
            }
            s = dot * a.scale;
            if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
            if (a.r1) s -= r1 * logf(1.f + r2 * (float)(pos - j));
        }
        float mx = s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_new = fmaxf(m, mx);
        if (m_new == -INFINITY) continue;
        const float alpha = expf(m - m_new), p = expf(s - m_new);
        m = m_new;
        float ps = p;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
        l = fmaf(l, alpha, ps);
#pragma unroll
        for (int i = 0; i < F32_MAX_DIM / 32; i++) acc[i] *= alpha;
        for (int t = 0; t < 32; t++) {
            const float pt = __shfl_sync(0xffffffffu, p, t);
            if (pt == 0.f) continue;  // the same for every lane
            const float* kt = key_row<float>(a.keys, rd.seq, j0 + t);
            if (!kt) continue;
            kt += (int64_t)kvh * D;
#pragma unroll
            for (int i = 0; i < F32_MAX_DIM / 32; i++)
                if (i * 32 + lane < D) acc[i] = fmaf(pt, kt[i * 32 + lane], acc[i]);
        }
    }
    const float f = (l > 0.f ? 1.f / l : 0.f) * (a.gate ? sigmoid(a.gate[(int64_t)row * a.n_q_heads + head]) : 1.f);
    float* out = reinterpret_cast<float*>(a.out) + (int64_t)row * a.out_stride + (int64_t)head * D;
#pragma unroll
    for (int i = 0; i < F32_MAX_DIM / 32; i++)
        if (i * 32 + lane < D) out[i * 32 + lane] = acc[i] * f;
}

template <int D, int MT, int SL>
cudaError_t launch_one(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    const int splits = wattn_splits(ctx, a, l, TOK, 16 * MT, SL == 1 ? 1 : MT == 1 ? 3 : 2);
    const WattnScratch sc = wattn_scratch(ctx, scratch);
    constexpr size_t smem = wattn_smem<D, MT, SL>();
    static SmemOptIn configured;
    if (cudaError_t e = tsb_opt_in_smem(ctx, window_attn_kernel<D, MT, SL>, smem, configured); e != cudaSuccess) return e;
    cudaError_t e = tsb_launch(ctx, window_attn_kernel<D, MT, SL>, dim3((unsigned)splits, (unsigned)a.keys.kv_heads, (unsigned)l.n_tiles), dim3(32 * MT * SL),
                               smem, st, true, a, l.tiles, l.tiles_per_group, l.rows_per_seq, l.rows_per_tile, sc.o, sc.ml, sc.tickets, ctx->dev_error);
    return e == cudaSuccess && splits > 1 ? launch_window_attn_merge(ctx, st, a, l, splits, 16 * MT, sc) : e;
}

template <int D, int NQ>
cudaError_t launch_few(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    using F = FewQ<D, NQ>;
    const int splits = wattn_splits(ctx, a, l, F::TILE, 8 * NQ, F::PER_SM);
    const WattnScratch sc = wattn_scratch(ctx, scratch);
    static SmemOptIn configured;
    if (cudaError_t e = tsb_opt_in_smem(ctx, window_attn_few_kernel<D, NQ>, F::SMEM, configured); e != cudaSuccess) return e;
    cudaError_t e = tsb_launch(ctx, window_attn_few_kernel<D, NQ>, dim3((unsigned)splits, (unsigned)a.keys.kv_heads, (unsigned)l.n_tiles), dim3(128), F::SMEM,
                               st, true, a, l.tiles, l.rows_per_seq, sc.o, sc.ml, sc.tickets, ctx->dev_error);
    return e == cudaSuccess && splits > 1 && NQ > 1 ? launch_window_attn_merge(ctx, st, a, l, splits, 8 * NQ, sc) : e;
}
// query tiles by the number of queries; head sizes above 128 have registers for one
template <int D>
cudaError_t launch_few_dim(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int queries, void* scratch) {
    if (queries <= 8) return launch_few<D, 1>(ctx, st, a, l, scratch);
    if (queries <= 16) return launch_one<D, 1, 4>(ctx, st, a, l, scratch);  // sixteen query rows of one mma tile: faster than two tiles of eight
    if constexpr (D <= 128) {
        if (queries <= 24) return launch_few<D, 3>(ctx, st, a, l, scratch);
        if (queries <= 32) return launch_few<D, 4>(ctx, st, a, l, scratch);
    }
    return launch_one<D, 4, 2>(ctx, st, a, l, scratch);
}

template <int MT, int SL>
cudaError_t launch_large(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, void* scratch) {
    switch (a.keys.head_dim) {
        case 32: return launch_one<32, MT, SL>(ctx, st, a, l, scratch);
        case 64: return launch_one<64, MT, SL>(ctx, st, a, l, scratch);
        case 96: return launch_one<96, MT, SL>(ctx, st, a, l, scratch);
        case 128: return launch_one<128, MT, SL>(ctx, st, a, l, scratch);
        case 192: return launch_one<192, MT, SL>(ctx, st, a, l, scratch);
        case 256: return launch_one<256, MT, SL>(ctx, st, a, l, scratch);
        default: return cudaErrorInvalidValue;
    }
}

cudaError_t launch_small(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int queries, void* scratch) {
    switch (a.keys.head_dim) {
        case 32: return launch_few_dim<32>(ctx, st, a, l, queries, scratch);
        case 64: return launch_few_dim<64>(ctx, st, a, l, queries, scratch);
        case 96: return launch_few_dim<96>(ctx, st, a, l, queries, scratch);
        case 128: return launch_few_dim<128>(ctx, st, a, l, queries, scratch);
        case 192: return launch_few_dim<192>(ctx, st, a, l, queries, scratch);
        case 256: return launch_few_dim<256>(ctx, st, a, l, queries, scratch);
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace

cudaError_t launch_window_attn_merge(tsb_ctx* ctx, cudaStream_t st, const WindowAttn& a, const WattnLaunch& l, int splits, int slots, const WattnScratch& sc) {
    return tsb_launch(ctx, window_attn_merge_kernel, dim3((unsigned)l.n_tiles, (unsigned)l.rows_per_tile, (unsigned)((a.n_q_heads + 7) / 8)), dim3(256), 0, st, true, a, l.tiles,
                      l.tiles_per_group, l.rows_per_seq, l.rows_per_tile, splits, slots, (const float*)sc.o, (const float2*)sc.ml);
}

size_t wattn_scratch_bytes(const tsb_ctx* ctx) {
    return WATTN_TICKETS * sizeof(uint32_t) + wattn_part_queries(ctx) * (sizeof(float2) + 256 * sizeof(float));
}

int wattn_rows_per_tile(int head_dim, int group) {
    const int per = WATTN_LARGE_Q / group > 0 ? WATTN_LARGE_Q / group : 1;
    return wattn_tc_supported(head_dim, group) ? 2 * per : per;
}

int wattn_pad_dim(int head_dim, bool f32) {
    if (head_dim <= 0) return 0;
    if (f32) return head_dim <= F32_MAX_DIM ? (head_dim + 3) / 4 * 4 : 0;
    for (int d : {32, 64, 96, 128, 192, 256})
        if (head_dim <= d) return d;
    return 0;
}

bool wattn_supported(int head_dim, int group, bool f32) { return wattn_pad_dim(head_dim, f32) > 0 && group >= 1 && (f32 || group <= WATTN_LARGE_Q); }

cudaError_t launch_window_attn(tsb_ctx* ctx, cudaStream_t st, bool f32, const WindowAttn& a, const AttnBatch& b, void* scratch) {
    if (f32)
        return tsb_launch(ctx, window_attn_f32_kernel, dim3((unsigned)(((int64_t)b.rows * a.n_q_heads + F32_WARPS - 1) / F32_WARPS)), dim3(F32_WARPS * 32),
                          0, st, true, a, b.rows, ctx->dev_error);
    const int grp = a.n_q_heads / a.keys.kv_heads, rpt = wattn_rows_per_tile(a.keys.head_dim, grp);
    auto large = [&](const WattnLaunch& l) {
        return wattn_tc_supported(a.keys.head_dim, grp) ? launch_window_attn_tc(ctx, st, a, l, scratch) : launch_large<8, 1>(ctx, st, a, l, scratch);
    };
    if (b.rows_per_seq > 0) {
        const int groups = b.rows / b.rows_per_seq, queries = b.rows_per_seq * grp;
        if (queries <= WATTN_SMALL_Q) return launch_small(ctx, st, a, WattnLaunch{nullptr, groups, 1, b.rows_per_seq, b.rows_per_seq, b.max_len}, queries, scratch);
        const int tpg = (b.rows_per_seq + rpt - 1) / rpt;
        return large(WattnLaunch{nullptr, groups * tpg, tpg, b.rows_per_seq, rpt, b.max_len});
    }
    cudaError_t e = cudaSuccess;
    if (b.n_large > 0) e = large(WattnLaunch{b.large, b.n_large, 1, 0, rpt, b.max_len});
    if (e == cudaSuccess && b.n_small > 0) e = launch_small(ctx, st, a, WattnLaunch{b.small, b.n_small, 1, 0, WATTN_SMALL_Q / grp, b.max_len}, b.small_queries, scratch);
    return e;
}
