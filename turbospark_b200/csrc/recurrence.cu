// Recurrent mixers row by row: decoded tokens, short portions, and every portion in f32.
//
// A CTA owns 32 value columns of one head of one portion; its slice of the state stays in registers over the portion's rows.  Eight
// lanes hold four columns each, the CTA's 32 such groups of lanes share out the state's rows (CR each).  Rows go through in batches of
// eight (or one by one where every portion is a row): their q, k, v and gates are brought to shared memory, every thread steps through the
// batch without a barrier and leaves its part of each output, then the parts are added.  Decays are applied as s + (decay - 1) s, with
// decay - 1 from expm1 or the gate itself: close to one the rounding of the factor would add up over a long memory.  A decoded token reads and
// writes the state once.
#include <algorithm>

#include "recurrence_dev.cuh"

namespace {

constexpr int THREADS = 256, COLS = REC_COLS, GROUPS = THREADS / 8;

template <int KIND, int BATCH>
size_t rows_smem(int dim_pad) {
    return ((size_t)BATCH * dim_pad * 2 + BATCH * COLS + (size_t)BATCH * GROUPS * COLS + (KIND == REC_MLSTM ? BATCH * GROUPS : 0) + 3 * BATCH) *
           sizeof(float);
}

// is the state after row t of the portion one of those that are kept?
__device__ __forceinline__ bool is_kept(const Recurrence& a, const AttnTile& p, int t) { return t + a.state.ring >= p.n_rows; }

template <typename T, int KIND, int CR, int BATCH>
__global__ void __launch_bounds__(THREADS) recurrence_rows_kernel(const __grid_constant__ Recurrence a, const __grid_constant__ RowTiles portions, uint32_t* __restrict__ err) {
    constexpr int DIM = GROUPS * CR;
    extern __shared__ __align__(16) float smem[];
    float *qs = smem, *ks = qs + BATCH * DIM, *vs = ks + BATCH * DIM;
    float *parts = vs + BATCH * COLS, *nparts = parts + BATCH * GROUPS * COLS, *decay = nparts + (KIND == REC_MLSTM ? BATCH * GROUPS : 0);
    float *write = decay + BATCH, *floor_ = write + BATCH;
    const int head = blockIdx.y, col0 = blockIdx.x * COLS;
    const int grp = threadIdx.x >> 3, vl = threadIdx.x & 7, c0 = grp * CR;
    const AttnTile p = row_tile(portions, blockIdx.z);
    const tsb_row_desc rd = a.rows[p.row_first];
    const int pos0 = rd.base + rd.slot, vp = recurrence_v_pitch(a.vdim), col = col0 + vl * 4;
    const bool ok = rd.seq >= 0 && rd.seq < a.state.n_streams;
    if (!ok) {
        if (threadIdx.x == 0) atomicCAS(err, 0u, (uint32_t)TSB_DEV_BAD_INDEX);
        pdl_wait();
        return;
    }
    // the state was written by an earlier pass
    float4 s[CR];
    float n[KIND == REC_MLSTM ? CR : 1];
    double top = 0.0;
    const int64_t head_state = (int64_t)a.dim * vp;
    {
        const int64_t at = (rec_slot(a, rd.seq, pos0 - 1) * a.heads + head);
        const float* p0 = a.state.s + at * head_state;
#pragma unroll
        for (int r = 0; r < CR; r++) {
            const bool in = pos0 > 0 && c0 + r < a.dim && col < vp;
            s[r] = in ? *reinterpret_cast<const float4*>(p0 + (int64_t)(c0 + r) * vp + col) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (KIND == REC_MLSTM) n[r] = pos0 > 0 && c0 + r < a.dim ? a.state.norm[(at * gridDim.x + blockIdx.x) * a.dim + c0 + r] : 0.f;
        }
        if (KIND == REC_MLSTM && pos0 > 0) top = a.state.top[at * gridDim.x + blockIdx.x];
    }
    const float rate = KIND == REC_SSD ? expf(a.a_log[head]) : 0.f, skip = KIND == REC_SSD ? a.skip[head] : 0.f;
    const int key_at = head / a.heads_per_key * a.dim;
    pdl_wait();
    pdl_launch_dependents();
    for (int b0 = 0; b0 < p.n_rows; b0 += BATCH) {
        const int nb = min(BATCH, p.n_rows - b0), row0 = p.row_first + b0;
        if (KIND != REC_FORGET) {
            if (threadIdx.x < nb) {
                const int t = threadIdx.x;
                const float2 g = KIND == REC_MLSTM ? mlstm_gates(a, row0 + t, head) : ssd_gates(a, row0 + t, head, rate);
                if (KIND == REC_SSD) write[t] = g.x, decay[t] = expm1f(g.y);
                else write[t] = g.x, decay[t] = g.y;
            }
            if (KIND == REC_MLSTM) {
                // the running maximum: every thread walks it, the first ones keep the factors
                __syncthreads();
                double m = top;
                float mine_w = 0.f, mine_d = 0.f, mine_m = 0.f;
                for (int t = 0; t < nb; t++) {
                    const double keep = (double)decay[t] + m, m_new = fmax(keep, (double)write[t]);
                    if (t == (int)threadIdx.x) {
                        mine_d = expm1f((float)(keep - m_new)), mine_w = expf((float)((double)write[t] - m_new)), mine_m = expf(-(float)m_new);
                        if (is_kept(a, p, b0 + t)) a.state.top[(rec_slot(a, rd.seq, pos0 + b0 + t) * a.heads + head) * gridDim.x + blockIdx.x] = m_new;
                    }
                    m = m_new;
                }
                __syncthreads();
                if (threadIdx.x < nb) decay[threadIdx.x] = mine_d, write[threadIdx.x] = mine_w, floor_[threadIdx.x] = mine_m;
                top = m;
            }
            __syncthreads();
        }
        for (int i = threadIdx.x; i < nb * DIM; i += THREADS) {
            const int t = i / DIM, c = i - t * DIM, row = row0 + t;
            float q = 0.f, k = 0.f;
            if (c < a.dim) {
                q = rec_get(static_cast<const T*>(a.q) + (int64_t)row * a.q_stride + key_at + c);
                if (KIND == REC_FORGET) {
                    const float l = a.lower[(int64_t)head * a.dim + c];
                    k = (1.f - l) * rec_sigmoid(-a.gate[(int64_t)row * a.gate_stride + (int64_t)head * a.dim + c]);  // 1 - f
                    q = rec_silu(q);
                } else {
                    k = rec_get(static_cast<const T*>(a.k) + (int64_t)row * a.k_stride + key_at + c) * write[t];
                    q *= a.q_scale;
                }
            }
            qs[i] = q, ks[i] = k;
        }
        for (int i = threadIdx.x; i < nb * COLS; i += THREADS) {
            const int t = i / COLS, c = col0 + i % COLS;
            vs[i] = c < a.vdim ? rec_get(static_cast<const T*>(a.v) + (int64_t)(row0 + t) * a.v_stride + (int64_t)head * a.vdim + c) : 0.f;
        }
        __syncthreads();
        for (int t = 0; t < nb; t++) {
            const float4 v = *reinterpret_cast<const float4*>(vs + t * COLS + vl * 4);
            const float dt = KIND == REC_FORGET ? 0.f : decay[t];
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
            float on = 0.f;
#pragma unroll
            for (int r = 0; r < CR; r++) {
                const float k = ks[t * DIM + c0 + r], q = qs[t * DIM + c0 + r];
                if (KIND == REC_FORGET) {  // f s + (1 - f) v
                    s[r].x = fmaf(k, v.x - s[r].x, s[r].x), s[r].y = fmaf(k, v.y - s[r].y, s[r].y);
                    s[r].z = fmaf(k, v.z - s[r].z, s[r].z), s[r].w = fmaf(k, v.w - s[r].w, s[r].w);
                } else {
                    s[r].x = fmaf(k, v.x, fmaf(dt, s[r].x, s[r].x)), s[r].y = fmaf(k, v.y, fmaf(dt, s[r].y, s[r].y));
                    s[r].z = fmaf(k, v.z, fmaf(dt, s[r].z, s[r].z)), s[r].w = fmaf(k, v.w, fmaf(dt, s[r].w, s[r].w));
                }
                o.x = fmaf(q, s[r].x, o.x), o.y = fmaf(q, s[r].y, o.y), o.z = fmaf(q, s[r].z, o.z), o.w = fmaf(q, s[r].w, o.w);
                if (KIND == REC_MLSTM) n[r] = fmaf(dt, n[r], n[r]) + k, on = fmaf(q, n[r], on);
            }
            *reinterpret_cast<float4*>(parts + (t * GROUPS + grp) * COLS + vl * 4) = o;
            if (KIND == REC_MLSTM && vl == 0) nparts[t * GROUPS + grp] = on;
            if (is_kept(a, p, b0 + t)) {
                const int64_t at = rec_slot(a, rd.seq, pos0 + b0 + t) * a.heads + head;
                float* dst = a.state.s + at * head_state;
#pragma unroll
                for (int r = 0; r < CR; r++) {
                    if (c0 + r >= a.dim) continue;
                    if (col < vp) *reinterpret_cast<float4*>(dst + (int64_t)(c0 + r) * vp + col) = s[r];
                    if (KIND == REC_MLSTM && vl == 0) a.state.norm[(at * gridDim.x + blockIdx.x) * a.dim + c0 + r] = n[r];
                }
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nb * COLS; i += THREADS) {
            const int t = i / COLS, c = i % COLS;
            float o = 0.f;
#pragma unroll 8
            for (int g = 0; g < GROUPS; g++) o += parts[(t * GROUPS + g) * COLS + c];
            if (KIND == REC_MLSTM) {
                float nq = 0.f;
#pragma unroll 8
                for (int g = 0; g < GROUPS; g++) nq += nparts[t * GROUPS + g];
                o /= fmaxf(fabsf(nq), floor_[t]) + 1e-6f;
            }
            if (KIND == REC_SSD) o = fmaf(skip, vs[i], o);
            if (col0 + c < a.vdim) a.out[(int64_t)(row0 + t) * a.out_stride + (int64_t)head * a.vdim + col0 + c] = o;
        }
        __syncthreads();
    }
}

template <typename T, int KIND, int CR, int BATCH>
cudaError_t launch_batch(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RowTiles& portions) {
    const size_t smem = rows_smem<KIND, BATCH>(GROUPS * CR);
    static SmemOptIn configured;
    if (smem > 48 * 1024)
        if (cudaError_t e = tsb_opt_in_smem(ctx, recurrence_rows_kernel<T, KIND, CR, BATCH>, smem, configured); e != cudaSuccess) return e;
    return tsb_launch(ctx, recurrence_rows_kernel<T, KIND, CR, BATCH>, dim3((unsigned)recurrence_copies(r.vdim), (unsigned)r.heads, (unsigned)portions.n), dim3(THREADS),
                      smem, st, true, r, portions, ctx->dev_error);
}
template <typename T, int KIND, int CR>
cudaError_t launch_rows(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RowTiles& portions) {
    if constexpr (sizeof(T) == 2 && CR <= 8)  // decoded tokens: little shared memory, more CTAs per SM
        if (portions.longest == 1) return launch_batch<T, KIND, CR, 1>(ctx, st, r, portions);
    return launch_batch<T, KIND, CR, 8>(ctx, st, r, portions);
}
template <typename T, int KIND>
cudaError_t launch_dim(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RowTiles& portions) {
    if (r.dim <= GROUPS * 2) return launch_rows<T, KIND, 2>(ctx, st, r, portions);
    if (r.dim <= GROUPS * 4) return launch_rows<T, KIND, 4>(ctx, st, r, portions);
    if (r.dim <= GROUPS * 8) return launch_rows<T, KIND, 8>(ctx, st, r, portions);
    return r.dim <= REC_MAX_DIM ? launch_rows<T, KIND, 32>(ctx, st, r, portions) : cudaErrorInvalidValue;
}
template <typename T>
cudaError_t launch_kind(tsb_ctx* ctx, cudaStream_t st, const Recurrence& r, const RowTiles& portions) {
    switch (r.kind) {
        case REC_FORGET: return launch_dim<T, REC_FORGET>(ctx, st, r, portions);
        case REC_MLSTM: return launch_dim<T, REC_MLSTM>(ctx, st, r, portions);
        case REC_SSD: return launch_dim<T, REC_SSD>(ctx, st, r, portions);
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace

cudaError_t launch_recurrence_rows(tsb_ctx* ctx, cudaStream_t st, bool f32, const Recurrence& r, const RowTiles& portions) {
    if (portions.n == 0) return cudaSuccess;
    return f32 ? launch_kind<float>(ctx, st, r, portions) : launch_kind<__nv_bfloat16>(ctx, st, r, portions);
}
