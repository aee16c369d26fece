// The matrix-memory recurrence 64 tokens at a time, bf16 projections, on mma.sync.  Within a chunk that starts from
// (S, n, m) the recurrence has a closed form.  With F_t the running sum of the log forget gates of the chunk,
//   m_t = F_t + max(m, max_{s<=t} (i_s - F_s)),     P_ts = (q_t . k_s) e^(F_t - F_s + i_s - m_t)  (s <= t)
//   o_t = [ e^(F_t + m - m_t) S^T q_t + sum_s P_ts v_s ] / (max(|e^(F_t + m - m_t) n.q_t + sum_s P_ts|, e^(-m_t)) + 1e-6)
// and the state moves to the chunk's end as S e^(F_L + m - m_L) + sum_s e^(F_L - F_s + i_s - m_L) k_s v_s^T.  Every exponent
// is at most zero.
//
// A CTA owns COLS value columns of one head of one sequence and walks the chunks; the state slice stays in registers as
// mma accumulators (f32).  What enters a product besides the projections themselves — S, P and the weighted values — is
// split into a bf16 head and remainder (two products), so state and weights keep about 16 bits on the tensor cores; their
// sums are f32.  Query, key and value tiles of the next chunk load (cp.async) while this one is computed.
#include "mlstm.cuh"

#include <algorithm>

namespace {

constexpr int CH_T = 256, CH_L = 64, CH_P_LD = CH_L + 8;

template <int COLS>
struct ChSmem {
    int ld;                                                // elements per q / k row
    size_t q, k, v, s_hi, s_lo, wv_hi, wv_lo, p_hi, p_lo, vec, total;
    static constexpr int kLdV = COLS + 8;
    static __host__ __device__ ChSmem of(int dim) {
        ChSmem s{};
        s.ld = dim + 8;
        const size_t qk = (size_t)CH_L * s.ld * 2, vt = (size_t)CH_L * kLdV * 2, st = (size_t)dim * kLdV * 2, pt = (size_t)CH_L * CH_P_LD * 2;
        s.q = 0;
        s.k = s.q + 2 * qk;
        s.v = s.k + 2 * qk;
        s.s_hi = s.v + 2 * vt;
        s.s_lo = s.s_hi + st;
        s.wv_hi = s.s_lo + st;
        s.wv_lo = s.wv_hi + vt;
        s.p_hi = s.wv_lo + vt;
        s.p_lo = s.p_hi + pt;
        s.vec = s.p_lo + pt;                               // f32: n [dim], F, w_in, w_up, x, m, nq, row sums [2] of 64 each, scalars
        s.total = s.vec + ((size_t)dim + 8 * CH_L + 8) * 4;
        return s;
    }
};

__device__ __forceinline__ void ch_cp16(uint32_t dst, const void* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void split_store(bf16* hi, bf16* lo, size_t at, float a, float b) {
    const uint32_t h = pack_bf16x2(a, b);
    *reinterpret_cast<uint32_t*>(hi + at) = h;
    *reinterpret_cast<uint32_t*>(lo + at) = pack_bf16x2(a - bf16_lo(h), b - bf16_hi(h));
}

// MTW: 16-row tiles of the state per warp (dim <= 128 * MTW)
template <int COLS, int MTW>
__global__ void __launch_bounds__(CH_T) mlstm_chunk_kernel(MlstmArgs a) {
    extern __shared__ __align__(128) unsigned char ch_smem[];
    using SM = ChSmem<COLS>;
    constexpr int NT = COLS / 8;                            // 8-column tiles of the slice
    constexpr int NO = NT / 2;                              // ... per warp in the output products (4 row tiles x 2 halves)
    const scr_mlstm_shape& s = a.s;
    const int dim = s.dim, vdim = s.vdim, H = s.heads;
    const SM lay = SM::of(dim);
    bf16* const Q = reinterpret_cast<bf16*>(ch_smem + lay.q);
    bf16* const K = reinterpret_cast<bf16*>(ch_smem + lay.k);
    bf16* const V = reinterpret_cast<bf16*>(ch_smem + lay.v);
    bf16 *s_hi = reinterpret_cast<bf16*>(ch_smem + lay.s_hi), *s_lo = reinterpret_cast<bf16*>(ch_smem + lay.s_lo);
    bf16 *wv_hi = reinterpret_cast<bf16*>(ch_smem + lay.wv_hi), *wv_lo = reinterpret_cast<bf16*>(ch_smem + lay.wv_lo);
    bf16 *p_hi = reinterpret_cast<bf16*>(ch_smem + lay.p_hi), *p_lo = reinterpret_cast<bf16*>(ch_smem + lay.p_lo);
    float* n = reinterpret_cast<float*>(ch_smem + lay.vec);
    float *F = n + dim, *w_in = F + CH_L, *w_up = w_in + CH_L, *gx = w_up + CH_L, *mt = gx + CH_L, *nq = mt + CH_L, *psum = nq + CH_L, *scal = psum + 2 * CH_L;
    pdl_trigger();
    const int c0 = blockIdx.x * COLS, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g = lane >> 2, t4 = lane & 3, lm = lane >> 3, lr = lane & 7;
    const int first = a.st.segs[b * 4], count = a.st.segs[b * 4 + 1], pos0 = a.st.segs[b * 4 + 2], slot = a.st.segs[b * 4 + 3];
    pdl_wait();
    if (count <= 0) return;
    if (slot < 0 || slot >= a.st.num_slots || first < 0 || first + count > a.st.rows) {
        if (tid == 0) atomicCAS(a.status, 0, SEQ_BAD_SLOT);
        return;
    }
    const size_t head = (size_t)slot * H + h;
    float* gs = a.state_s + head * dim * vdim;
    const int slices = mlstm_slices(vdim), slice0 = c0 / SCR_MLSTM_SLICE, nslice = min(COLS / SCR_MLSTM_SLICE, slices - slice0);
    float* gn = a.state_n + (head * slices + slice0) * dim;
    float* gm = a.state_m + head * slices + slice0;
    const bool fresh = pos0 == 0;
    const bf16* proj = reinterpret_cast<const bf16*>(a.proj);
    const int qchunks = dim / 8, chunks = (count + CH_L - 1) / CH_L;
    auto load_chunk = [&](int c) {
        const int st = c & 1;
        for (int i = tid; i < CH_L * qchunks * 2; i += CH_T) {
            const int which = i / (CH_L * qchunks), e = i - which * CH_L * qchunks, r = e / qchunks, x = e - r * qchunks;
            const bool ok = c * CH_L + r < count;
            const bf16* src = proj + (size_t)(first + (ok ? c * CH_L + r : 0)) * a.ld + (size_t)(which ? H + h : h) * dim + x * 8;
            ch_cp16(smem_u32((which ? K : Q) + (size_t)st * CH_L * lay.ld + (size_t)r * lay.ld + x * 8), src, ok);
        }
        for (int i = tid; i < CH_L * NT; i += CH_T) {
            const int r = i / NT, x = i - r * NT;
            const bool ok = c * CH_L + r < count && c0 + x * 8 < vdim;
            const bf16* src = proj + (size_t)(first + (ok ? c * CH_L + r : 0)) * a.ld + (size_t)2 * H * dim + (size_t)h * vdim + (ok ? c0 + x * 8 : 0);
            ch_cp16(smem_u32(V + (size_t)st * CH_L * SM::kLdV + (size_t)r * SM::kLdV + x * 8), src, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_chunk(0);

    // state slice: warp w holds rows (w * MTW + m) * 16 .. + 16 as accumulators
    float S[MTW][NT][4];
#pragma unroll
    for (int m = 0; m < MTW; ++m)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = (warp * MTW + m) * 16 + g + (e >> 1) * 8, c = c0 + nt * 8 + t4 * 2 + (e & 1);
                S[m][nt][e] = (!fresh && r < dim && c < vdim) ? gs[(size_t)r * vdim + c] : 0.0f;
            }
    for (int i = tid; i < dim; i += CH_T) n[i] = fresh ? 0.0f : gn[i];
    float m_run = fresh ? 0.0f : gm[0];
    const float qscale = 1.0f / sqrtf(float(dim));

    for (int c = 0; c < chunks; ++c) {
        const int len = min(CH_L, count - c * CH_L), st = c & 1;
        const bf16 *Qc = Q + (size_t)st * CH_L * lay.ld, *Kc = K + (size_t)st * CH_L * lay.ld, *Vc = V + (size_t)st * CH_L * SM::kLdV;
        // the state of the chunk's start as matrix operands
#pragma unroll
        for (int m = 0; m < MTW; ++m) {
            const int r = (warp * MTW + m) * 16 + g;
            if ((warp * MTW + m) * 16 >= dim) break;
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) {
                split_store(s_hi, s_lo, (size_t)r * SM::kLdV + nt * 8 + t4 * 2, S[m][nt][0], S[m][nt][1]);
                split_store(s_hi, s_lo, (size_t)(r + 8) * SM::kLdV + nt * 8 + t4 * 2, S[m][nt][2], S[m][nt][3]);
            }
        }
        if (warp == 0) {                                   // gates: two tokens per lane, prefix sums and maxima over the warp
            float f[2], gi[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = lane * 2 + e, row = first + c * CH_L + t;
                f[e] = t < len ? mlstm_gate_f(a, row, h) : 0.0f;           // past the end: nothing is forgotten or written
                gi[e] = t < len ? mlstm_gate_i(a, row, h) : -INFINITY;
            }
            float run = f[0] + f[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, run, o);
                if (lane >= o) run += up;
            }
            const float F1 = run, F0 = run - f[1];
            const float x0 = gi[0] - F0, x1 = gi[1] - F1;
            float best = fmaxf(x0, x1);
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, best, o);
                if (lane >= o) best = fmaxf(best, up);
            }
            float before = __shfl_up_sync(0xffffffffu, best, 1);
            if (lane == 0) before = -INFINITY;
            const float m0 = F0 + fmaxf(m_run, fmaxf(before, x0)), m1 = F1 + fmaxf(m_run, best);
            F[lane * 2] = F0;
            F[lane * 2 + 1] = F1;
            gx[lane * 2] = x0;
            gx[lane * 2 + 1] = x1;
            mt[lane * 2] = m0;
            mt[lane * 2 + 1] = m1;
            w_in[lane * 2] = expf(F0 + m_run - m0);
            w_in[lane * 2 + 1] = expf(F1 + m_run - m1);
            const float FL = __shfl_sync(0xffffffffu, F1, 31), mL = __shfl_sync(0xffffffffu, m1, 31);
            w_up[lane * 2] = expf(FL + x0 - mL);
            w_up[lane * 2 + 1] = expf(FL + x1 - mL);
            if (lane == 0) {
                scal[0] = mL;
                scal[1] = expf(FL + m_run - mL);
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (c + 1 < chunks) load_chunk(c + 1);
        const float m_next = scal[0], keep = scal[1];

        // P = (Q K^T) with weights: warp = (16-row tile, half of the keys)
        const int rt = warp & 3, half = warp >> 2;
        {
            float p[4][4] = {};
            const uint32_t qa = smem_u32(Qc + (size_t)(rt * 16 + (lm & 1) * 8 + lr) * lay.ld + (lm >> 1) * 8);
            const uint32_t kb = smem_u32(Kc + (size_t)(half * 32 + (lm >> 1) * 8 + lr) * lay.ld + (lm & 1) * 8);
            if (half * 32 <= rt * 16 + 15)                 // (the other tiles lie above the diagonal)
                for (int ks = 0; ks < dim / 16; ++ks) {
                    uint32_t qf[4];
                    ldsm_x4(qa + ks * 32, qf);
#pragma unroll
                    for (int n2 = 0; n2 < 2; ++n2) {
                        uint32_t kf[4];
                        ldsm_x4(kb + (uint32_t)(n2 * 16 * lay.ld * 2) + ks * 32, kf);
                        mma_16816(p[n2 * 2], qf[0], qf[1], qf[2], qf[3], kf[0], kf[1]);
                        mma_16816(p[n2 * 2 + 1], qf[0], qf[1], qf[2], qf[3], kf[2], kf[3]);
                    }
                }
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int t = rt * 16 + g + hf * 8;
                const float base = F[t] - mt[t];
                float sum = 0.0f;
#pragma unroll
                for (int nt = 0; nt < 4; ++nt) {
                    const int key = half * 32 + nt * 8 + t4 * 2;
                    const float e0 = key <= t ? p[nt][hf * 2] * qscale * expf(base + gx[key]) : 0.0f;
                    const float e1 = key + 1 <= t ? p[nt][hf * 2 + 1] * qscale * expf(base + gx[key + 1]) : 0.0f;
                    sum += e0 + e1;
                    split_store(p_hi, p_lo, (size_t)t * CH_P_LD + key, e0, e1);
                }
                sum += __shfl_xor_sync(0xffffffffu, sum, 1);
                sum += __shfl_xor_sync(0xffffffffu, sum, 2);
                if (t4 == 0) psum[half * CH_L + t] = sum;
            }
        }
        {                                                  // n . q: four threads per token
            const int t = tid >> 2, part = tid & 3;
            float d = 0.0f;
            for (int i = part * 2; i < dim; i += 8) {
                const uint32_t w = *reinterpret_cast<const uint32_t*>(Qc + (size_t)t * lay.ld + i);
                d = fmaf(bf16_lo(w), n[i], fmaf(bf16_hi(w), n[i + 1], d));
            }
            d += __shfl_xor_sync(0xffffffffu, d, 1);
            d += __shfl_xor_sync(0xffffffffu, d, 2);
            if (part == 0) nq[t] = d * qscale * w_in[t];
        }
        for (int i = tid; i < CH_L * COLS / 2; i += CH_T) {  // values weighted for the state's update
            const int r = i / (COLS / 2), x = (i - r * (COLS / 2)) * 2;
            const uint32_t w = *reinterpret_cast<const uint32_t*>(Vc + (size_t)r * SM::kLdV + x);
            split_store(wv_hi, wv_lo, (size_t)r * SM::kLdV + x, bf16_lo(w) * w_up[r], bf16_hi(w) * w_up[r]);
        }
        __syncthreads();

        // O = w_in q^T S + P V: warp = (16-row tile, half of the columns)
        {
            float o[NO][4] = {};
            const uint32_t qa = smem_u32(Qc + (size_t)(rt * 16 + (lm & 1) * 8 + lr) * lay.ld + (lm >> 1) * 8);
            for (int ks = 0; ks < dim / 16; ++ks) {
                uint32_t qf[4];
                ldsm_x4(qa + ks * 32, qf);
#pragma unroll
                for (int n2 = 0; n2 < NO / 2; ++n2) {
                    const size_t at = (size_t)(ks * 16 + (lm & 1) * 8 + lr) * SM::kLdV + half * (COLS / 2) + n2 * 16 + (lm >> 1) * 8;
                    uint32_t bh[4], bl[4];
                    ldsm_x4_trans(smem_u32(s_hi + at), bh);
                    ldsm_x4_trans(smem_u32(s_lo + at), bl);
                    mma_16816(o[n2 * 2], qf[0], qf[1], qf[2], qf[3], bh[0], bh[1]);
                    mma_16816(o[n2 * 2 + 1], qf[0], qf[1], qf[2], qf[3], bh[2], bh[3]);
                    mma_16816(o[n2 * 2], qf[0], qf[1], qf[2], qf[3], bl[0], bl[1]);
                    mma_16816(o[n2 * 2 + 1], qf[0], qf[1], qf[2], qf[3], bl[2], bl[3]);
                }
            }
            const int t0 = rt * 16 + g;
            const float u0 = w_in[t0] * qscale, u1 = w_in[t0 + 8] * qscale;
#pragma unroll
            for (int x = 0; x < NO; ++x) {
                o[x][0] *= u0;
                o[x][1] *= u0;
                o[x][2] *= u1;
                o[x][3] *= u1;
            }
            for (int ks = 0; ks <= rt; ++ks) {              // keys past the row tile weigh nothing
                uint32_t ph[4], pl[4];
                const size_t pat = (size_t)(rt * 16 + (lm & 1) * 8 + lr) * CH_P_LD + ks * 16 + (lm >> 1) * 8;
                ldsm_x4(smem_u32(p_hi + pat), ph);
                ldsm_x4(smem_u32(p_lo + pat), pl);
#pragma unroll
                for (int n2 = 0; n2 < NO / 2; ++n2) {
                    uint32_t vf[4];
                    ldsm_x4_trans(smem_u32(Vc + (size_t)(ks * 16 + (lm & 1) * 8 + lr) * SM::kLdV + half * (COLS / 2) + n2 * 16 + (lm >> 1) * 8), vf);
                    mma_16816(o[n2 * 2], ph[0], ph[1], ph[2], ph[3], vf[0], vf[1]);
                    mma_16816(o[n2 * 2 + 1], ph[0], ph[1], ph[2], ph[3], vf[2], vf[3]);
                    mma_16816(o[n2 * 2], pl[0], pl[1], pl[2], pl[3], vf[0], vf[1]);
                    mma_16816(o[n2 * 2 + 1], pl[0], pl[1], pl[2], pl[3], vf[2], vf[3]);
                }
            }
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int t = t0 + hf * 8;
                if (t >= len) continue;
                const float inv = 1.0f / (fmaxf(fabsf(nq[t] + psum[t] + psum[CH_L + t]), expf(-mt[t])) + 1e-6f);
                float* dst = a.out + (size_t)(first + c * CH_L + t) * H * vdim + (size_t)h * vdim;
#pragma unroll
                for (int x = 0; x < NO; ++x) {
                    const int col = c0 + half * (COLS / 2) + x * 8 + t4 * 2;
                    if (col < vdim) *reinterpret_cast<float2*>(dst + col) = make_float2(o[x][hf * 2] * inv, o[x][hf * 2 + 1] * inv);
                }
            }
        }
        // S <- keep S + K^T (weighted values); n likewise
#pragma unroll
        for (int m = 0; m < MTW; ++m) {
            const int r0 = (warp * MTW + m) * 16;
            if (r0 >= dim) break;
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[m][nt][e] *= keep;
#pragma unroll
            for (int ks = 0; ks < CH_L / 16; ++ks) {
                uint32_t kf[4];                             // A = K^T: rows are dimensions, columns tokens
                ldsm_x4_trans(smem_u32(Kc + (size_t)(ks * 16 + (lm >> 1) * 8 + lr) * lay.ld + r0 + (lm & 1) * 8), kf);
#pragma unroll
                for (int n2 = 0; n2 < NT / 2; ++n2) {
                    const size_t at = (size_t)(ks * 16 + (lm & 1) * 8 + lr) * SM::kLdV + n2 * 16 + (lm >> 1) * 8;
                    uint32_t bh[4], bl[4];
                    ldsm_x4_trans(smem_u32(wv_hi + at), bh);
                    ldsm_x4_trans(smem_u32(wv_lo + at), bl);
                    mma_16816(S[m][n2 * 2], kf[0], kf[1], kf[2], kf[3], bh[0], bh[1]);
                    mma_16816(S[m][n2 * 2 + 1], kf[0], kf[1], kf[2], kf[3], bh[2], bh[3]);
                    mma_16816(S[m][n2 * 2], kf[0], kf[1], kf[2], kf[3], bl[0], bl[1]);
                    mma_16816(S[m][n2 * 2 + 1], kf[0], kf[1], kf[2], kf[3], bl[2], bl[3]);
                }
            }
        }
        for (int i = tid; i < dim; i += CH_T) {
            float v = keep * n[i];
#pragma unroll 8
            for (int r = 0; r < CH_L; ++r) v = fmaf(w_up[r], __bfloat162float(Kc[(size_t)r * lay.ld + i]), v);
            n[i] = v;
        }
        m_run = m_next;
        __syncthreads();                                   // before the next chunk rewrites S operands, gates and P
    }
#pragma unroll
    for (int m = 0; m < MTW; ++m)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int r = (warp * MTW + m) * 16 + g + (e >> 1) * 8, cc = c0 + nt * 8 + t4 * 2;
                if (r < dim && cc < vdim) *reinterpret_cast<float2*>(gs + (size_t)r * vdim + cc) = make_float2(S[m][nt][e], S[m][nt][e + 1]);
            }
    for (int sl = 0; sl < nslice; ++sl) {
        for (int i = tid; i < dim; i += CH_T) gn[(size_t)sl * dim + i] = n[i];
        if (tid == 0) gm[sl] = m_run;
    }
}

template <int COLS, int MTW>
cudaError_t ch_launch(const MlstmArgs& a, cudaStream_t stream) {
    const size_t smem = ChSmem<COLS>::of(a.s.dim).total;
    const cudaError_t e = seq_smem(mlstm_chunk_kernel<COLS, MTW>, smem);
    if (e != cudaSuccess) return e;
    return launch_pdl(mlstm_chunk_kernel<COLS, MTW>, dim3(scr_ceil_div(a.s.vdim, COLS), a.s.heads, a.st.batch), dim3(CH_T), smem, stream, a);
}

}  // namespace

bool mlstm_chunk_applies(const scr_mlstm_shape& s, const scr_step& st) {
    return st.max_count >= 8 && s.dim % 16 == 0 && s.dim <= 256 && s.vdim % 8 == 0;
}

int32_t mlstm_chunk_launch(scr_ctx* ctx, const MlstmArgs& a, cudaStream_t stream) {
    if (a.ld % 8 || !scr_aligned16(a.proj)) return scr_fail(ctx, SCR_E_ALIGN, "mlstm projections need 16-byte rows");
    // narrow slices while they fit the GPU in one round (the chunks of a head are a chain), and where the wide ones do not fit an SM
    const bool narrow = a.s.dim > 128 || a.s.vdim <= 32 || scr_ceil_div(a.s.vdim, 32) * a.s.heads * a.st.batch <= ctx->sm_count;
    cudaError_t e;
    if (a.s.dim > 128) e = ch_launch<32, 2>(a, stream);
    else e = narrow ? ch_launch<32, 1>(a, stream) : ch_launch<64, 1>(a, stream);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "mlstm_chunk: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "mlstm_chunk");
}
