// Recurrent mixers over long portions, REC_CHUNK rows at a time, bfloat16 operands on mma.sync with f32 accumulators.
//
// With E_t the product of a chunk's decays up to row t and S the state before the chunk,
//   o_t = E_t q_t . S + sum_{s <= t} (E_t / E_s) (q_t . k_s) v_s,    S' = E_T S + sum_s (E_T / E_s) k_s v_s^T.
// A CTA owns VB value columns of one head of one portion and walks its chunks.  Four warps make the outputs - sixteen rows each: queries
// against the state, then against the chunk's keys, weights, values - while four others hold the state in their accumulators, bring it
// to the end of the chunk and leave it in shared memory for the next one.
//
// What is f32 stays f32-like: an operand that is not a projection (state, weighted products, decayed queries, keys or values) goes into a
// product as the sum of two bfloat16 numbers, which keeps 16 bits of it.
//
// Decay per head (REC_MLSTM, REC_SSD): E is a number per row; the ratios are exponentials of differences of its logarithm, applied to the
// products of plain queries and keys.
// Decay per row of the state (REC_FORGET): E is a vector; queries times E_t and keys over E_s are made per chunk.  The keys grow as E falls,
// so a chunk is cut where a component of E falls below 2^-80 and goes on from there (rows outside the cut are zero).
#include <algorithm>

#include "mma_dev.cuh"
#include "recurrence_dev.cuh"

namespace {

constexpr int C = REC_CHUNK, THREADS = 256;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float E_MIN = 8.2718061e-25f;  // 2^-80

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ uint32_t pack(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
// two numbers as the sum of two bfloat16 pairs
__device__ __forceinline__ void split(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack(a, b);
    lo = pack(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xFFFF0000u));
}
// byte offset of 16-byte piece p of row r; rows of BYTES, pieces permuted so that eight rows' worth of one piece spread over all banks
template <int BYTES>
__device__ __forceinline__ uint32_t at(int r, int p) {
    return (uint32_t)(r * BYTES + ((BYTES == 64 ? (p ^ ((r >> 1) & 3)) : (p ^ (r & 7))) << 4));
}

template <int KIND, int DK, int VB>
struct Smem {
    static constexpr int KEY = C * DK * 2, VAL = C * VB * 2, STATE = DK * VB * 2;
    static constexpr bool FORGET = KIND == REC_FORGET;
    // FORGET: queries and keys, each high and low part, made per chunk; else two stages of queries and keys as they come
    static constexpr int Q = 0, K = FORGET ? 2 * KEY : KEY, KEY_STAGE = 2 * KEY;
    static constexpr int V = 4 * KEY;                 // two stages
    static constexpr int W = V + 2 * VAL;             // weighted values, high and low (not FORGET)
    static constexpr int S = W + (FORGET ? 0 : 2 * VAL);  // two states, high and low each
    static constexpr int Z = S + 4 * STATE;           // FORGET: pre-activations (f32) and queries as they come
    static constexpr int RAW_Q = Z + C * DK * 4;
    static constexpr int F = FORGET ? RAW_Q + KEY : Z;  // f32 vectors
    static constexpr int N_F = FORGET ? 2 * DK + THREADS : 5 * C + 8 + 2 * DK;
    static constexpr int BYTES = F + N_F * 4;
};

template <int KIND, int DK, int VB>
__global__ void __launch_bounds__(THREADS, 1)
    recurrence_chunks_kernel(const __grid_constant__ Recurrence a, const __grid_constant__ RowTiles portions, uint32_t* __restrict__ err) {
    using M = Smem<KIND, DK, VB>;
    constexpr bool FORGET = KIND == REC_FORGET, MLSTM = KIND == REC_MLSTM, SSD = KIND == REC_SSD;
    constexpr int KS = DK / 16, NV = VB / 8, MS = DK / 64, KB = DK * 2, BV = VB * 2;
    constexpr int RS = FORGET ? THREADS / DK : 1, TR = C / RS;  // FORGET: a thread makes queries and keys of one channel and TR rows
    extern __shared__ __align__(128) uint8_t smem[];
    const uint32_t base = smem_u32(smem);
    float* fv = reinterpret_cast<float*>(smem + M::F);
    // decay per head: row factor and exponents per row, scalars of the chunk
    float *ea = fv, *eb = fv + C, *gain = fv + 2 * C, *floor_ = fv + 3 * C, *wv = fv + 4 * C, *scal = fv + 5 * C, *norm = scal + 8;
    // decay per channel: E at the end of the cut, lower bounds, products of the row splits
    float *e_end = fv, *lower = fv + DK, *totals = fv + 2 * DK;
    __shared__ int cut_end;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int head = blockIdx.y, col0 = blockIdx.x * VB, vp = recurrence_v_pitch(a.vdim);
    const AttnTile p = row_tile(portions, blockIdx.z);
    const tsb_row_desc rd = a.rows[p.row_first];
    const int pos0 = rd.base + rd.slot, key_at = head / a.heads_per_key * a.dim;
    if (rd.seq < 0 || rd.seq >= a.state.n_streams) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        pdl_wait();
        return;
    }
    const int n_chunks = (p.n_rows + C - 1) / C;
    const __nv_bfloat16 *gq = static_cast<const __nv_bfloat16*>(a.q) + key_at, *gk = static_cast<const __nv_bfloat16*>(a.k) + key_at;
    const __nv_bfloat16* gv = static_cast<const __nv_bfloat16*>(a.v) + (int64_t)head * a.vdim + col0;

    // ---- copies of a chunk (rows and columns outside are zeros)
    auto issue = [&](int chunk) {
        if (chunk < n_chunks) {
            const int row0 = p.row_first + chunk * C, n = min(C, p.n_rows - chunk * C), st = chunk & 1;
            if (!FORGET) {
                for (int i = threadIdx.x; i < C * (DK / 8); i += THREADS) {
                    const int r = i / (DK / 8), c = i % (DK / 8);
                    const bool ok = r < n && c * 8 < a.dim;
                    const int64_t row = ok ? row0 + r : row0, col = ok ? c * 8 : 0;
                    cp16(base + st * M::KEY_STAGE + M::Q + at<KB>(r, c), gq + row * a.q_stride + col, ok);
                    cp16(base + st * M::KEY_STAGE + M::K + at<KB>(r, c), gk + row * a.k_stride + col, ok);
                }
            }
            for (int i = threadIdx.x; i < C * (VB / 8); i += THREADS) {
                const int r = i / (VB / 8), c = i % (VB / 8);
                const bool ok = r < n && col0 + c * 8 < a.vdim;
                cp16(base + M::V + st * M::VAL + at<BV>(r, c), gv + (int64_t)(ok ? row0 + r : row0) * a.v_stride + (ok ? c * 8 : 0), ok);
            }
        }
        cp_async_commit();
    };
    const int ch = threadIdx.x % DK, split_i = threadIdx.x / DK;  // FORGET: the thread's channel and rows
    auto z_at = [&](int r) -> float& { return reinterpret_cast<float*>(smem + M::Z)[r * DK + ch]; };
    auto raw = [&](int chunk) {  // FORGET: pre-activations and queries of a chunk
        if (!FORGET || chunk >= n_chunks) return;
        const int row0 = p.row_first + chunk * C, n = min(C, p.n_rows - chunk * C);
        const float* gz = a.gate + (int64_t)head * a.dim;
        for (int i = threadIdx.x; i < C * (DK / 4); i += THREADS) {
            const int r = i / (DK / 4), c = i % (DK / 4);
            const bool ok = r < n && c * 4 < a.dim;
            cp16(base + M::Z + (r * DK + c * 4) * 4, gz + (ok ? row0 + r : row0) * a.gate_stride + (ok ? c * 4 : 0), ok);
        }
        for (int i = threadIdx.x; i < C * (DK / 8); i += THREADS) {
            const int r = i / (DK / 8), c = i % (DK / 8);
            const bool ok = r < n && c * 8 < a.dim;
            cp16(base + M::RAW_Q + (r * DK + c * 8) * 2, gq + (int64_t)(ok ? row0 + r : row0) * a.q_stride + (ok ? c * 8 : 0), ok);
        }
    };
    // decay per head: lane l of warp 0 has the gates of rows 2 l and 2 l + 1 of the next chunk
    float2 gate2[2];
    const float rate = SSD ? expf(a.a_log[head]) : 0.f;
    auto fetch_gates = [&](int chunk) {
        if (FORGET || warp != 0 || chunk >= n_chunks) return;
        const int n = min(C, p.n_rows - chunk * C);
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int r = 2 * lane + i, row = p.row_first + chunk * C + r;
            gate2[i] = r < n ? (MLSTM ? mlstm_gates(a, row, head) : ssd_gates(a, row, head, rate)) : make_float2(MLSTM ? -1e30f : 0.f, 0.f);
        }
    };

    // ---- the state before the portion, written by an earlier pass: accumulators of warps 4 .. 7, m-tiles warp - 4, warp, ..
    float s[MS][NV][4];
    double top = 0.0;
    const int64_t head_state = (int64_t)a.dim * vp;
    const int64_t slot0 = rec_slot(a, rd.seq, pos0 - 1) * a.heads + head;
    auto state_to_smem = [&](int buf) {
#pragma unroll
        for (int m = 0; m < MS; m++)
#pragma unroll
            for (int n = 0; n < NV; n++)
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const int r = (warp - 4 + 4 * m) * 16 + gid + 8 * h;
                    uint32_t hi, lo;
                    split(s[m][n][2 * h], s[m][n][2 * h + 1], hi, lo);
                    const uint32_t off = at<BV>(r, n) + tig * 4;
                    *reinterpret_cast<uint32_t*>(smem + M::S + 2 * buf * M::STATE + off) = hi;
                    *reinterpret_cast<uint32_t*>(smem + M::S + (2 * buf + 1) * M::STATE + off) = lo;
                }
    };
    if (warp >= 4) {
        const float* src = a.state.s + slot0 * head_state;
#pragma unroll
        for (int m = 0; m < MS; m++)
#pragma unroll
            for (int n = 0; n < NV; n++)
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const int r = (warp - 4 + 4 * m) * 16 + gid + 8 * (i >> 1), c = col0 + n * 8 + 2 * tig + (i & 1);
                    s[m][n][i] = pos0 > 0 && r < a.dim && c < vp ? src[(int64_t)r * vp + c] : 0.f;
                }
        state_to_smem(0);
        if (MLSTM)
            for (int i = threadIdx.x - 128; i < DK; i += 128) norm[i] = pos0 > 0 && i < a.dim ? a.state.norm[slot0 * a.dim + i] : 0.f;
    }
    if (MLSTM && pos0 > 0) top = a.state.top[slot0];
    const float skip = SSD ? a.skip[head] : 0.f;
    if (FORGET)
        for (int i = threadIdx.x; i < DK; i += THREADS) lower[i] = i < a.dim ? a.lower[(int64_t)head * a.dim + i] : 1.f;
    pdl_wait();
    raw(0);
    issue(0);
    fetch_gates(0);

    int state_buf = 0;
    for (int chunk = 0; chunk < n_chunks; chunk++) {
        const int n = min(C, p.n_rows - chunk * C), row0 = p.row_first + chunk * C;
        if (!FORGET) issue(chunk + 1), cp_async_wait<1>();
        else cp_async_wait<0>();
        if (!FORGET && warp == 0) {
            const float d0 = gate2[0].y, d1 = gate2[1].y;
            float sum = d0 + d1;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float v = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += v;
            }
            const float l1 = sum, l0 = sum - d1;  // log decay up to rows 2 lane + 1 and 2 lane
            const float l_end = __shfl_sync(0xffffffffu, sum, 31);
            if (SSD) {
                ea[2 * lane] = l0 * LOG2E, ea[2 * lane + 1] = l1 * LOG2E, eb[2 * lane] = -l0 * LOG2E, eb[2 * lane + 1] = -l1 * LOG2E;
                gain[2 * lane] = gate2[0].x, gain[2 * lane + 1] = gate2[1].x;
                if (lane == 0) scal[0] = l_end * LOG2E, scal[1] = expf(l_end);
            } else {
                // relative to the maximum before the chunk: i_s - F_s - m, and its running maximum with 0
                const float b0 = (float)((double)gate2[0].x - l0 - top), b1 = (float)((double)gate2[1].x - l1 - top);
                float mx = fmaxf(b0, b1);
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const float v = __shfl_up_sync(0xffffffffu, mx, o);
                    if (lane >= o) mx = fmaxf(mx, v);
                }
                const float before = __shfl_up_sync(0xffffffffu, mx, 1);
                const float m1 = fmaxf(mx, 0.f), m0 = fmaxf(lane > 0 ? fmaxf(before, b0) : b0, 0.f), m_end = __shfl_sync(0xffffffffu, m1, 31);
                ea[2 * lane] = -m0 * LOG2E, ea[2 * lane + 1] = -m1 * LOG2E, eb[2 * lane] = b0 * LOG2E, eb[2 * lane + 1] = b1 * LOG2E;
                gain[2 * lane] = gain[2 * lane + 1] = 1.f;
                floor_[2 * lane] = expf(-(float)(top + l0 + m0)), floor_[2 * lane + 1] = expf(-(float)(top + l1 + m1));
                if (lane == 0) scal[0] = -m_end * LOG2E, scal[1] = expf(-m_end);
                top += (double)l_end + m_end;
            }
            fetch_gates(chunk + 1);
        }
        __syncthreads();  // the chunk's copies and gates are there
        const uint32_t vt = base + M::V + (chunk & 1) * M::VAL;

        for (int cut = 0; cut < n;) {  // FORGET: usually once
            int end = n;
            if (FORGET) {
                // E from row `cut` on: products within the thread's rows, then over the row splits.  The first time round the pre-activations
                // become 1 - f = (1 - l) sigmoid(-z).
                const float low = lower[ch];
                float mine = 1.f;
#pragma unroll 4
                for (int i = 0; i < TR; i++) {
                    const int r = split_i * TR + i;
                    float& x = z_at(r);
                    if (cut == 0) {
                        const float e = __expf(-fabsf(x)), d = __fdividef(1.f, 1.f + e);
                        x = r < n ? (1.f - low) * (x >= 0.f ? e * d : d) : 0.f;
                    }
                    if (r >= cut) mine *= 1.f - x;
                }
                totals[threadIdx.x] = mine;
                if (threadIdx.x == 0) cut_end = n;
                __syncthreads();
                float e0 = 1.f;
                for (int i = 0; i < split_i; i++) e0 *= totals[i * DK + ch];
                // E only falls: the chunk is cut if it ends too low
                if (__syncthreads_or(e0 * mine < E_MIN)) {
                    float e = e0;
                    for (int i = 0; i < TR; i++) {
                        const int r = split_i * TR + i;
                        if (r < cut || r >= n) continue;
                        e *= 1.f - z_at(r);
                        if (e < E_MIN && r > cut) {
                            atomicMin(&cut_end, r);
                            break;
                        }
                    }
                    __syncthreads();
                    end = cut_end;
                }
                float e = e0;
#pragma unroll 4
                for (int i = 0; i < TR; i++) {
                    const int r = split_i * TR + i;
                    const bool in = r >= cut && r < end;
                    const float k = z_at(r), x = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(smem + M::RAW_Q)[r * DK + ch]);
                    if (in) e = fmaxf(e * (1.f - k), E_MIN);  // the first row of a cut may fall further: nothing of the rows before is left then
                    const float qe = in ? __fdividef(x, 1.f + __expf(-x)) * e : 0.f, ke = in ? k * (1.f / e) : 0.f;
                    const __nv_bfloat16 qh = __float2bfloat16_rn(qe), kh = __float2bfloat16_rn(ke);
                    const uint32_t off = at<KB>(r, ch >> 3) + (ch & 7) * 2;
                    *reinterpret_cast<__nv_bfloat16*>(smem + M::Q + off) = qh;
                    *reinterpret_cast<__nv_bfloat16*>(smem + M::Q + M::KEY + off) = __float2bfloat16_rn(qe - __bfloat162float(qh));
                    *reinterpret_cast<__nv_bfloat16*>(smem + M::K + off) = kh;
                    *reinterpret_cast<__nv_bfloat16*>(smem + M::K + M::KEY + off) = __float2bfloat16_rn(ke - __bfloat162float(kh));
                }
                if (end > split_i * TR && end <= (split_i + 1) * TR) e_end[ch] = e;
            } else {
                // values weighted to the end of the chunk
                for (int i = threadIdx.x; i < C * (VB / 2); i += THREADS) {
                    const int r = i / (VB / 2), c = i % (VB / 2);
                    const uint32_t off = at<BV>(r, c >> 2) + (c & 3) * 4;
                    const uint32_t v = *reinterpret_cast<const uint32_t*>(smem + M::V + (chunk & 1) * M::VAL + off);
                    const float w = ex2(scal[0] + eb[r]) * gain[r];
                    if (MLSTM && c == 0) wv[r] = w;
                    uint32_t hi, lo;
                    split(__uint_as_float(v << 16) * w, __uint_as_float(v & 0xFFFF0000u) * w, hi, lo);
                    *reinterpret_cast<uint32_t*>(smem + M::W + off) = hi;
                    *reinterpret_cast<uint32_t*>(smem + M::W + M::VAL + off) = lo;
                }
            }
            __syncthreads();
            if (FORGET && end == n) raw(chunk + 1), issue(chunk + 1);  // what they overwrite has been used
            const uint32_t qt = base + (FORGET ? 0 : (chunk & 1) * M::KEY_STAGE) + M::Q, kt = base + (FORGET ? 0 : (chunk & 1) * M::KEY_STAGE) + M::K;
            const uint32_t sh = base + M::S + 2 * state_buf * M::STATE, sl = sh + M::STATE;
            if (warp < 4) {
                // ---- outputs of rows 16 warp .. + 15
                const int t0 = warp * 16;
                if (t0 < end && t0 + 16 > cut) {
                    uint32_t qa[KS][4], ql[FORGET ? KS : 1][4];
#pragma unroll
                    for (int ks = 0; ks < KS; ks++) {
                        ldsm4(qa[ks], qt + at<KB>(t0 + (lane & 15), ks * 2 + (lane >> 4)));
                        if (FORGET) ldsm4(ql[FORGET ? ks : 0], qt + M::KEY + at<KB>(t0 + (lane & 15), ks * 2 + (lane >> 4)));
                    }
                    float o[NV][4];
#pragma unroll
                    for (int i = 0; i < NV; i++)
#pragma unroll
                        for (int j = 0; j < 4; j++) o[i][j] = 0.f;
#pragma unroll
                    for (int ks = 0; ks < KS; ks++)
#pragma unroll
                        for (int np = 0; np < NV / 2; np++) {
                            uint32_t bh[4], bl[4];
                            ldsm4_t(bh, sh + at<BV>(ks * 16 + (lane & 15), np * 2 + (lane >> 4)));
                            ldsm4_t(bl, sl + at<BV>(ks * 16 + (lane & 15), np * 2 + (lane >> 4)));
                            mma_bf16(o[2 * np], qa[ks], bh[0], bh[1]), mma_bf16(o[2 * np + 1], qa[ks], bh[2], bh[3]);
                            mma_bf16(o[2 * np], qa[ks], bl[0], bl[1]), mma_bf16(o[2 * np + 1], qa[ks], bl[2], bl[3]);
                            if (FORGET) mma_bf16(o[2 * np], ql[FORGET ? ks : 0], bh[0], bh[1]), mma_bf16(o[2 * np + 1], ql[FORGET ? ks : 0], bh[2], bh[3]);
                        }
                    const int ta = t0 + gid, tb = ta + 8;
                    const float ea0 = FORGET ? 0.f : ea[ta], ea1 = FORGET ? 0.f : ea[tb];
                    float nq[2] = {0.f, 0.f};  // MLSTM: the lane's share of n . q
                    if (!FORGET) {
                        const float f0 = ex2(ea0), f1 = ex2(ea1);
#pragma unroll
                        for (int i = 0; i < NV; i++) o[i][0] *= f0, o[i][1] *= f0, o[i][2] *= f1, o[i][3] *= f1;
                        if (MLSTM) {
                            const float* nb = norm + state_buf * DK;
#pragma unroll
                            for (int ks = 0; ks < KS; ks++) {
                                const float2 n0 = *reinterpret_cast<const float2*>(nb + ks * 16 + 2 * tig), n1 = *reinterpret_cast<const float2*>(nb + ks * 16 + 8 + 2 * tig);
#pragma unroll
                                for (int h = 0; h < 2; h++) {
                                    const uint32_t x = qa[ks][h], y = qa[ks][2 + h];
                                    nq[h] = fmaf(__uint_as_float(x << 16), n0.x, fmaf(__uint_as_float(x & 0xFFFF0000u), n0.y, nq[h]));
                                    nq[h] = fmaf(__uint_as_float(y << 16), n1.x, fmaf(__uint_as_float(y & 0xFFFF0000u), n1.y, nq[h]));
                                }
                            }
                            nq[0] *= f0, nq[1] *= f1;
                        }
                    }
                    for (int jt = cut / 16; jt <= warp; jt++) {
                        float s0[2][4];
#pragma unroll
                        for (int i = 0; i < 2; i++)
#pragma unroll
                            for (int j = 0; j < 4; j++) s0[i][j] = 0.f;
#pragma unroll
                        for (int kp = 0; kp < KS / 2; kp++)
#pragma unroll
                            for (int i = 0; i < 2; i++) {
                                uint32_t b[4];
                                ldsm4(b, kt + at<KB>(jt * 16 + i * 8 + (lane & 7), kp * 4 + (lane >> 3)));
                                mma_bf16(s0[i], qa[2 * kp], b[0], b[1]), mma_bf16(s0[i], qa[2 * kp + 1], b[2], b[3]);
                                if (FORGET) {
                                    uint32_t bl[4];
                                    ldsm4(bl, kt + M::KEY + at<KB>(jt * 16 + i * 8 + (lane & 7), kp * 4 + (lane >> 3)));
                                    mma_bf16(s0[i], qa[2 * kp], bl[0], bl[1]), mma_bf16(s0[i], qa[2 * kp + 1], bl[2], bl[3]);
                                    mma_bf16(s0[i], ql[FORGET ? 2 * kp : 0], b[0], b[1]), mma_bf16(s0[i], ql[FORGET ? 2 * kp + 1 : 0], b[2], b[3]);
                                }
                            }
                        uint32_t ph[4], pl[4];
#pragma unroll
                        for (int i = 0; i < 2; i++) {
                            const int c0 = jt * 16 + i * 8 + 2 * tig;
#pragma unroll
                            for (int j = 0; j < 4; j++) {
                                const int c = c0 + (j & 1), t = j < 2 ? ta : tb;
                                float w = 0.f;
                                if (c <= t) w = FORGET ? s0[i][j] : s0[i][j] * (ex2((j < 2 ? ea0 : ea1) + eb[c]) * gain[c]);
                                s0[i][j] = w;
                            }
                            if (MLSTM) nq[0] += s0[i][0] + s0[i][1], nq[1] += s0[i][2] + s0[i][3];
                            split(s0[i][0], s0[i][1], ph[2 * i], pl[2 * i]);
                            split(s0[i][2], s0[i][3], ph[2 * i + 1], pl[2 * i + 1]);
                        }
#pragma unroll
                        for (int np = 0; np < NV / 2; np++) {
                            uint32_t b[4];
                            ldsm4_t(b, vt + at<BV>(jt * 16 + (lane & 15), np * 2 + (lane >> 4)));
                            mma_bf16(o[2 * np], ph, b[0], b[1]), mma_bf16(o[2 * np + 1], ph, b[2], b[3]);
                            mma_bf16(o[2 * np], pl, b[0], b[1]), mma_bf16(o[2 * np + 1], pl, b[2], b[3]);
                        }
                    }
                    float out_f[2] = {a.q_scale, a.q_scale};
                    if (MLSTM) {
#pragma unroll
                        for (int h = 0; h < 2; h++) {
                            nq[h] += __shfl_xor_sync(0xffffffffu, nq[h], 1);
                            nq[h] += __shfl_xor_sync(0xffffffffu, nq[h], 2);
                            out_f[h] = a.q_scale / (fmaxf(fabsf(nq[h] * a.q_scale), floor_[h ? tb : ta]) + 1e-6f);
                        }
                    }
#pragma unroll
                    for (int h = 0; h < 2; h++) {
                        const int t = h ? tb : ta;
                        if (t < cut || t >= end) continue;
                        float* dst = a.out + (int64_t)(row0 + t) * a.out_stride + (int64_t)head * a.vdim + col0;
#pragma unroll
                        for (int i = 0; i < NV; i++) {
                            float2 v = make_float2(o[i][2 * h] * out_f[h], o[i][2 * h + 1] * out_f[h]);
                            if (SSD) {
                                const uint32_t x = *reinterpret_cast<const uint32_t*>(smem + M::V + (chunk & 1) * M::VAL + at<BV>(t, i) + tig * 4);
                                v.x = fmaf(skip, __uint_as_float(x << 16), v.x), v.y = fmaf(skip, __uint_as_float(x & 0xFFFF0000u), v.y);
                            }
                            if (col0 + i * 8 + 2 * tig < a.vdim) *reinterpret_cast<float2*>(dst + i * 8 + 2 * tig) = v;
                        }
                    }
                }
            } else {
                // ---- the state at the end of the chunk (or of the cut)
                if (!FORGET) {
                    const float d = scal[1];
#pragma unroll
                    for (int m = 0; m < MS; m++)
#pragma unroll
                        for (int i = 0; i < NV; i++)
#pragma unroll
                            for (int j = 0; j < 4; j++) s[m][i][j] *= d;
                }
                const uint32_t bh_at = FORGET ? vt : base + M::W;
                for (int ks = cut / 16; ks * 16 < end; ks++) {
                    uint32_t bh[NV / 2][4], bl[FORGET ? 1 : NV / 2][4];
#pragma unroll
                    for (int np = 0; np < NV / 2; np++) {
                        ldsm4_t(bh[np], bh_at + at<BV>(ks * 16 + (lane & 15), np * 2 + (lane >> 4)));
                        if (!FORGET) ldsm4_t(bl[FORGET ? 0 : np], bh_at + M::VAL + at<BV>(ks * 16 + (lane & 15), np * 2 + (lane >> 4)));
                    }
#pragma unroll
                    for (int m = 0; m < MS; m++) {
                        const int c8 = (warp - 4 + 4 * m) * 2 + ((lane >> 3) & 1), r = ks * 16 + (lane & 7) + ((lane >> 4) << 3);
                        uint32_t ka[4], kl[4];
                        ldsm4_t(ka, kt + at<KB>(r, c8));
                        if (FORGET) ldsm4_t(kl, kt + M::KEY + at<KB>(r, c8));
#pragma unroll
                        for (int np = 0; np < NV / 2; np++) {
                            mma_bf16(s[m][2 * np], ka, bh[np][0], bh[np][1]), mma_bf16(s[m][2 * np + 1], ka, bh[np][2], bh[np][3]);
                            if (FORGET) {
                                mma_bf16(s[m][2 * np], kl, bh[np][0], bh[np][1]), mma_bf16(s[m][2 * np + 1], kl, bh[np][2], bh[np][3]);
                            } else {
                                const uint32_t(&x)[4] = bl[FORGET ? 0 : np];
                                mma_bf16(s[m][2 * np], ka, x[0], x[1]), mma_bf16(s[m][2 * np + 1], ka, x[2], x[3]);
                            }
                        }
                    }
                }
                if (FORGET) {
#pragma unroll
                    for (int m = 0; m < MS; m++) {
                        const float d0 = e_end[(warp - 4 + 4 * m) * 16 + gid], d1 = e_end[(warp - 4 + 4 * m) * 16 + gid + 8];
#pragma unroll
                        for (int i = 0; i < NV; i++) s[m][i][0] *= d0, s[m][i][1] *= d0, s[m][i][2] *= d1, s[m][i][3] *= d1;
                    }
                }
                state_to_smem(state_buf ^ 1);
                if (MLSTM) {
                    for (int c = threadIdx.x - 128; c < DK; c += 128) {
                        float x = norm[state_buf * DK + c] * scal[1];
#pragma unroll 8
                        for (int r = 0; r < C; r++)
                            x = fmaf(wv[r], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(
                                                               smem + (chunk & 1) * M::KEY_STAGE + M::K + at<KB>(r, c >> 3) + (c & 7) * 2)), x);
                        norm[(state_buf ^ 1) * DK + c] = x;
                    }
                }
            }
            state_buf ^= 1;
            cut = end;
            __syncthreads();  // outputs have read what the next cut or chunk overwrites
        }
    }
    cp_async_wait<0>();
    pdl_launch_dependents();
    const int64_t slot = rec_slot(a, rd.seq, pos0 + p.n_rows - 1) * a.heads + head;
    if (warp >= 4) {
        float* dst = a.state.s + slot * head_state;
#pragma unroll
        for (int m = 0; m < MS; m++)
#pragma unroll
            for (int n = 0; n < NV; n++)
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const int r = (warp - 4 + 4 * m) * 16 + gid + 8 * h, c = col0 + n * 8 + 2 * tig;
                    if (r < a.dim && c < vp) *reinterpret_cast<float2*>(dst + (int64_t)r * vp + c) = make_float2(s[m][n][2 * h], s[m][n][2 * h + 1]);
                }
        if (MLSTM && blockIdx.x == 0)
            for (int i = threadIdx.x - 128; i < a.dim; i += 128) a.state.norm[slot * a.dim + i] = norm[state_buf * DK + i];
    }
    if (MLSTM && blockIdx.x == 0 && threadIdx.x == 0) a.state.top[slot] = top;
}

template <int KIND, int DK, int VB>
cudaError_t launch_chunks(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RowTiles& portions) {
    constexpr size_t smem = Smem<KIND, DK, VB>::BYTES;
    static_assert(smem <= 226 * 1024, "");
    static SmemOptIn configured;
    if (cudaError_t e = tsb_opt_in_smem(ctx, recurrence_chunks_kernel<KIND, DK, VB>, smem, configured); e != cudaSuccess) return e;
    return tsb_launch(ctx, recurrence_chunks_kernel<KIND, DK, VB>, dim3((unsigned)((r.vdim + VB - 1) / VB), (unsigned)r.heads, (unsigned)portions.n), dim3(THREADS), smem,
                      st, true, r, portions, ctx->dev_error);
}
template <int KIND>
cudaError_t launch_chunks_dim(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RowTiles& portions) {
    if (r.dim <= 64) return launch_chunks<KIND, 64, 32>(ctx, st, r, portions);
    if constexpr (KIND != REC_FORGET)
        if (r.dim > 128) return launch_chunks<KIND, 256, 32>(ctx, st, r, portions);
    return launch_chunks<KIND, 128, 32>(ctx, st, r, portions);
}

}  // namespace

bool recurrence_chunks_supported(int kind, int dim, int vdim) { return dim <= (kind == REC_FORGET ? 128 : 256) && dim % 8 == 0 && vdim % 8 == 0; }

cudaError_t launch_recurrence_chunks(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RowTiles& portions) {
    if (portions.n == 0) return cudaSuccess;
    switch (r.kind) {
        case REC_FORGET: return launch_chunks_dim<REC_FORGET>(ctx, st, r, portions);
        case REC_MLSTM: return launch_chunks_dim<REC_MLSTM>(ctx, st, r, portions);
        case REC_SSD: return launch_chunks_dim<REC_SSD>(ctx, st, r, portions);
        default: return cudaErrorInvalidValue;
    }
}
