// Matrix-memory recurrences 64 tokens at a time, bf16 projections, on mma.sync: the mLSTM (mlstm_chunk.cu), and the memory with
// a constant decay (DECAY, lightning_chunk.cu).  Within a chunk of the mLSTM that starts from
// (S, n, m) the recurrence has a closed form.  With F_t the running sum of the log forget gates of the chunk,
//   m_t = F_t + max(m, max_{s<=t} (i_s - F_s)),     P_ts = (q_t . k_s) e^(F_t - F_s + i_s - m_t)  (s <= t)
//   o_t = [ e^(F_t + m - m_t) S^T q_t + sum_s P_ts v_s ] / (max(|e^(F_t + m - m_t) n.q_t + sum_s P_ts|, e^(-m_t)) + 1e-6)
// and the state moves to the chunk's end as S e^(F_L + m - m_L) + sum_s e^(F_L - F_s + i_s - m_L) k_s v_s^T.  Every exponent
// is at most zero.  With a constant decay d and no normaliser the same form has P_ts = (q_t . k_s) d^(t - s),
// o_t = d^(t + 1) S^T q_t + sum_s P_ts v_s and S d^L + sum_s d^(L - 1 - s) k_s v_s^T, its powers from a table.
//
// A CTA owns COLS value columns of one head of one sequence and walks chunks; the state slice stays in registers as mma
// accumulators (f32), with the normaliser n as one more column (its "values" are ones).  What enters a product besides the
// projections themselves — S, P and the weighted values — is split into a bf16 head and remainder (two products), so
// state and weights keep about 16 bits on the tensor cores; their sums are f32.  Sixteen warps compute; one more sums up
// the gates of the next chunk meanwhile (their values come from a small kernel before).  Query, key and value tiles of the next chunk load (cp.async) while this one is
// computed.
//
// The chunks of a head are a chain.  Where heads and slices do not fill the GPU, a long sequence is cut into groups of
// chunks: a first launch runs only the state updates of every group (the first from the sequence's state, the others from
// nothing), a second one lets every group put together the state it starts from (S' = e^(F+m-m') S + e^(M-m') U over the
// groups before it) and compute its outputs; its last group leaves the sequence's state.
#pragma once

#include "memory.cuh"

#include <algorithm>

namespace {

constexpr int CH_WARPS = 16, CH_T = CH_WARPS * 32, CH_THREADS = CH_T + 32, CH_L = 64, CH_P_LD = CH_L + 8;
enum ChMode { CH_WHOLE, CH_STATES, CH_OUTPUTS };

// How a step is cut, and where the groups' states go: per (sequence, head, slice) entries 0 .. groups of
// [state fragments | n fragments | F, M]; entry 0 is the state the sequence starts from, entry g + 1 what group g leaves.
struct ChGroups {
    float* ws;
    int groups, chunks;                                    // groups per sequence, chunks per group
};

// RTILES: 16-row tiles of the state the warps cover (dim <= 16 * RTILES); the other warps share the slice's columns.
template <int COLS, int RTILES>
struct ChShape {
    static constexpr int kSplit = CH_WARPS / RTILES, kTiles = COLS / 8 / kSplit;      // column shares; 8-column tiles per warp
    static constexpr int kFrag = kTiles * 4, kEntryFloats = (kFrag + 2) * CH_T + 2;
    static_assert(kSplit * RTILES == CH_WARPS && kTiles * kSplit * 8 == COLS, "warps cover the state slice");
};

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
        s.vec = s.p_lo + pt;                               // f32: two sets of gates (F, w_in, w_up, x, m; scalars), row sums [4]
        s.total = s.vec + (2 * (5 * (size_t)CH_L + 4) + 4 * CH_L) * 4;
        return s;
    }
};

__device__ __forceinline__ void split_store(bf16* hi, bf16* lo, size_t at, float a, float b) {
    const uint32_t h = pack_bf16x2(a, b);
    *reinterpret_cast<uint32_t*>(hi + at) = h;
    *reinterpret_cast<uint32_t*>(lo + at) = pack_bf16x2(a - bf16_lo(h), b - bf16_hi(h));
}
__device__ __forceinline__ void ldsm_x2_trans(uint32_t addr, uint32_t& a, uint32_t& b) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(a), "=r"(b) : "r"(addr));
}

template <int COLS, int RTILES, ChMode MODE, bool DECAY>
__global__ void __launch_bounds__(CH_THREADS, 1) memory_chunk_kernel(MemoryArgs a, ChGroups gr) {
    extern __shared__ __align__(128) unsigned char ch_smem[];
    using SM = ChSmem<COLS>;
    using Shape = ChShape<COLS, RTILES>;
    constexpr int NTS = Shape::kTiles;                      // state: this warp's 8-column tiles
    constexpr int NO = COLS / 32;                           // outputs: 8-column tiles of a quarter of the columns
    constexpr int LDV = SM::kLdV, ENTRY = Shape::kEntryFloats;
    constexpr bool OUT = MODE != CH_STATES;
    const scr_mlstm_shape& s = a.s;
    const int dim = s.dim, vdim = s.vdim, H = s.heads;
    const SM lay = SM::of(dim);
    bf16* const Q = reinterpret_cast<bf16*>(ch_smem + lay.q);
    bf16* const K = reinterpret_cast<bf16*>(ch_smem + lay.k);
    bf16* const V = reinterpret_cast<bf16*>(ch_smem + lay.v);
    bf16 *s_hi = reinterpret_cast<bf16*>(ch_smem + lay.s_hi), *s_lo = reinterpret_cast<bf16*>(ch_smem + lay.s_lo);
    bf16 *wv_hi = reinterpret_cast<bf16*>(ch_smem + lay.wv_hi), *wv_lo = reinterpret_cast<bf16*>(ch_smem + lay.wv_lo);
    bf16 *p_hi = reinterpret_cast<bf16*>(ch_smem + lay.p_hi), *p_lo = reinterpret_cast<bf16*>(ch_smem + lay.p_lo);
    float* const sets = reinterpret_cast<float*>(ch_smem + lay.vec);
    constexpr int SET = 5 * CH_L + 4;
    float* const psum = sets + 2 * SET;                     // [quarter of the keys][token]
    pdl_trigger();
    const int c0 = blockIdx.x * COLS, h = blockIdx.y, b = blockIdx.z / gr.groups, grp = blockIdx.z - b * gr.groups;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, lm = lane >> 3, lr = lane & 7;
    const bool worker = warp < CH_WARPS;
    const int first = a.st.segs[b * 4], count = a.st.segs[b * 4 + 1], pos0 = a.st.segs[b * 4 + 2], slot = a.st.segs[b * 4 + 3];
    const int chunks = (count + CH_L - 1) / CH_L, c_lo = grp * gr.chunks, c_hi = min(c_lo + gr.chunks, chunks);
    const int last_grp = (chunks - 1) / gr.chunks;
    pdl_wait();
    if (count <= 0 || c_lo >= chunks || (MODE == CH_STATES && grp > 0 && grp == last_grp)) return;
    if (slot < 0 || slot >= a.st.num_slots || first < 0 || first + count > a.st.rows) {
        if (tid == 0) atomicCAS(a.status, 0, SEQ_BAD_SLOT);
        return;
    }
    const size_t head = (size_t)slot * H + h;
    float* gs = a.state_s + head * dim * vdim;
    const int slices = mlstm_slices(vdim), slice0 = c0 / SCR_MLSTM_SLICE, nslice = min(COLS / SCR_MLSTM_SLICE, slices - slice0);
    float* gn = DECAY ? nullptr : a.state_n + (head * slices + slice0) * dim;
    float* gm = DECAY ? nullptr : a.state_m + head * slices + slice0;
    float* entries = MODE == CH_WHOLE ? nullptr : gr.ws + (((size_t)b * H + h) * gridDim.x + blockIdx.x) * (gr.groups + 1) * ENTRY;
    const bool fresh = pos0 == 0;
    const bf16* proj = reinterpret_cast<const bf16*>(a.proj);
    const int qchunks = dim / 8;
    auto load_chunk = [&](int c) {                          // a warp per row: its query and key pieces, then its values
        if (!worker) return;
        const int st = c & 1;
#pragma unroll
        for (int i = 0; i < CH_L / CH_WARPS; ++i) {
            const int r = warp * (CH_L / CH_WARPS) + i;
            const bool ok = c * CH_L + r < count;
            const bf16* row = proj + (size_t)(first + (ok ? c * CH_L + r : 0)) * a.ld;
            for (int x = lane + (OUT ? 0 : qchunks); x < 2 * qchunks; x += 32) {
                const bool key = x >= qchunks;
                const int e = (key ? x - qchunks : x) * 8;
                cp_async16(smem_u32((key ? K : Q) + (size_t)(st * CH_L + r) * lay.ld + e), row + (size_t)(key ? H + h : h) * dim + e, ok);
            }
            if (lane < COLS / 8) {
                const bool in = ok && c0 + lane * 8 < vdim;
                cp_async16(smem_u32(V + (size_t)(st * CH_L + r) * LDV + lane * 8), row + (size_t)2 * H * dim + (size_t)h * vdim + (in ? c0 + lane * 8 : 0), in);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_chunk(c_lo);

    // state slice: rows r0 .. r0 + 16, columns col0 .. as accumulators; n in the first column's lanes of the warps that own column 0
    const int r0 = (warp % RTILES) * 16, col0 = (warp / RTILES) * NTS * 8;
    const bool mine = worker && r0 < dim, owns_n = !DECAY && mine && col0 == 0;
    // f_sum: the group's log decay, with a constant decay its factor
    float S[NTS][4], n[4] = {0.0f, 0.0f, 0.0f, 0.0f}, m_run = 0.0f, f_sum = DECAY ? 1.0f : 0.0f;
#pragma unroll
    for (int nt = 0; nt < NTS; ++nt) S[nt][0] = S[nt][1] = S[nt][2] = S[nt][3] = 0.0f;
    auto put_entry = [&](float* e) {
        if (worker) {
#pragma unroll
            for (int i = 0; i < NTS * 4; ++i) e[i * CH_T + tid] = S[i >> 2][i & 3];
            e[NTS * 4 * CH_T + tid] = n[0];
            e[(NTS * 4 + 1) * CH_T + tid] = n[2];
        } else if (lane == 0) {                             // (the gate warp knows the sums)
            e[ENTRY - 2] = f_sum;
            e[ENTRY - 1] = m_run;
        }
    };
    if (MODE == CH_OUTPUTS) {
        // entry 0, or for a later group what group 0 leaves, is a whole state; what the other groups leave joins it
        for (int e = grp == 0 ? 0 : 1; e <= grp; ++e) {
            const float* src = entries + (size_t)e * ENTRY;
            const float F = src[ENTRY - 2], M = src[ENTRY - 1];
            const bool whole = e <= 1;
            const float mn = whole ? M : fmaxf(F + m_run, M);
            const float keep = whole ? 0.0f : DECAY ? F : expf(F + m_run - mn), put = whole || DECAY ? 1.0f : expf(M - mn);
            m_run = mn;
            if (worker) {
#pragma unroll
                for (int i = 0; i < NTS * 4; ++i) S[i >> 2][i & 3] = keep * S[i >> 2][i & 3] + put * src[i * CH_T + tid];
                n[0] = keep * n[0] + put * src[NTS * 4 * CH_T + tid];
                n[2] = keep * n[2] + put * src[(NTS * 4 + 1) * CH_T + tid];
            }
        }
    } else if (grp == 0) {
        if (!fresh) {
            if (!DECAY) m_run = gm[0];
            if (mine) {
#pragma unroll
                for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int c = c0 + col0 + nt * 8 + t4 * 2 + (e & 1);
                        if (c < vdim) S[nt][e] = gs[(size_t)(r0 + g + (e >> 1) * 8) * vdim + c];
                    }
                if (owns_n && t4 == 0) {
                    n[0] = gn[r0 + g];
                    n[2] = gn[r0 + g + 8];
                }
            }
        }
        if (MODE == CH_STATES) {
            put_entry(entries);
            if (last_grp == 0) return;
        }
    } else {
        m_run = DECAY ? 0.0f : -INFINITY;                   // nothing remembered
    }
    const float qscale = DECAY ? 1.0f : 1.0f / sqrtf(float(dim));
    const float* pw = DECAY ? a.powers + (size_t)h * SCR_DECAY_POWERS : nullptr;
    // zero the columns beside the slice (the normaliser's tile) of the state's and the weighted values' operands once
    for (int i = tid; i < (dim + CH_L) * 4; i += CH_THREADS) {
        const int r = i >> 2, x = COLS + (i & 3) * 2;
        bf16 *hi = r < dim ? s_hi + (size_t)r * LDV : wv_hi + (size_t)(r - dim) * LDV, *lo = r < dim ? s_lo + (size_t)r * LDV : wv_lo + (size_t)(r - dim) * LDV;
        *reinterpret_cast<uint32_t*>(hi + x) = 0;
        *reinterpret_cast<uint32_t*>(lo + x) = 0;
    }
    __syncthreads();
    float next_f[2], next_i[2];                             // log gates of the next chunk, two tokens per lane
    auto fetch = [&](int c) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            if (DECAY) continue;
            const int t = c * CH_L + lane * 2 + e;
            const float* z = a.gates + (size_t)(first + t) * a.ld_gates + h;
            next_i[e] = t < count ? z[0] : -INFINITY;       // past the end: nothing is written or forgotten
            next_f[e] = t < count ? z[H] : 0.0f;
        }
    };
    // Gates of chunk c into their set, by one warp: two tokens per lane, prefix sums and maxima over the warp.
    auto gates = [&](int c) {
        float* F = sets + (c & 1) * SET;
        if (DECAY) {                                        // F: d^t; weights of the state and of the values
            const int len = min(CH_L, count - c * CH_L);
            float *w_in = F + CH_L, *w_up = w_in + CH_L, *scal = w_up + 3 * CH_L;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = lane * 2 + e;
                F[t] = pw[t];
                w_in[t] = pw[t + 1];
                w_up[t] = t < len ? pw[len - 1 - t] : 0.0f;
            }
            if (lane == 0) scal[0] = pw[len];
            f_sum *= pw[len];
            return;
        }
        float f[2] = {next_f[0], next_f[1]}, gi[2] = {next_i[0], next_i[1]};
        fetch(c + 1);
        float run = f[0] + f[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, o);
            if (lane >= o) run += up;
        }
        const float F1 = run, F0 = run - f[1], x0 = gi[0] - F0, x1 = gi[1] - F1;
        float best = fmaxf(x0, x1);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, best, o);
            if (lane >= o) best = fmaxf(best, up);
        }
        float before = __shfl_up_sync(0xffffffffu, best, 1);
        if (lane == 0) before = -INFINITY;
        const float m0 = F0 + fmaxf(m_run, fmaxf(before, x0)), m1 = F1 + fmaxf(m_run, best);
        const float FL = __shfl_sync(0xffffffffu, F1, 31), mL = __shfl_sync(0xffffffffu, m1, 31);
        float *w_in = F + CH_L, *w_up = w_in + CH_L, *gx = w_up + CH_L, *mt = gx + CH_L, *scal = mt + CH_L;
        *reinterpret_cast<float2*>(F + lane * 2) = make_float2(F0, F1);
        *reinterpret_cast<float2*>(w_in + lane * 2) = make_float2(expf(F0 + m_run - m0), expf(F1 + m_run - m1));
        *reinterpret_cast<float2*>(w_up + lane * 2) = make_float2(expf(FL + x0 - mL), expf(FL + x1 - mL));
        *reinterpret_cast<float2*>(gx + lane * 2) = make_float2(x0, x1);
        *reinterpret_cast<float2*>(mt + lane * 2) = make_float2(m0, m1);
        if (lane == 0) scal[0] = expf(FL + m_run - mL);
        m_run = mL;
        f_sum += FL;
    };
    if (!worker) {
        fetch(c_lo);
        gates(c_lo);
    }

    const int rt = warp & 3, quarter = (warp >> 2) & 3;     // P and O: 16-row tile, quarter of the keys / columns
    for (int c = c_lo; c < c_hi; ++c) {
        const int len = min(CH_L, count - c * CH_L), st = c & 1;
        const float *F = sets + (c & 1) * SET, *w_in = F + CH_L, *w_up = w_in + CH_L, *gx = w_up + CH_L, *mt = gx + CH_L, *scal = mt + CH_L;
        const bf16 *Qc = Q + (size_t)st * CH_L * lay.ld, *Kc = K + (size_t)st * CH_L * lay.ld, *Vc = V + (size_t)st * CH_L * LDV;
        if (OUT && mine) {                                  // the state of the chunk's start as matrix operands
            const size_t at = (size_t)(r0 + g) * LDV + col0 + t4 * 2;
#pragma unroll
            for (int nt = 0; nt < NTS; ++nt) {
                split_store(s_hi, s_lo, at + nt * 8, S[nt][0], S[nt][1]);
                split_store(s_hi, s_lo, at + 8 * LDV + nt * 8, S[nt][2], S[nt][3]);
            }
            if (owns_n && t4 == 0) {
                split_store(s_hi, s_lo, (size_t)(r0 + g) * LDV + COLS, n[0], 0.0f);
                split_store(s_hi, s_lo, (size_t)(r0 + g + 8) * LDV + COLS, n[2], 0.0f);
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (c + 1 < c_hi) load_chunk(c + 1);
        if (!worker) {
            if (c + 1 < c_hi) gates(c + 1);
        } else {
            if (OUT && quarter <= rt) {                     // P = (Q K^T) with weights (the other tiles lie above the diagonal)
                float p[2][4] = {};
                const uint32_t qa = smem_u32(Qc + (size_t)(rt * 16 + (lm & 1) * 8 + lr) * lay.ld + (lm >> 1) * 8);
                const uint32_t kb = smem_u32(Kc + (size_t)(quarter * 16 + (lm >> 1) * 8 + lr) * lay.ld + (lm & 1) * 8);
#pragma unroll 4
                for (int ks = 0; ks < dim / 16; ++ks) {
                    uint32_t qf[4], kf[4];
                    ldsm_x4(qa + ks * 32, qf);
                    ldsm_x4(kb + ks * 32, kf);
                    mma_16816(p[0], qf[0], qf[1], qf[2], qf[3], kf[0], kf[1]);
                    mma_16816(p[1], qf[0], qf[1], qf[2], qf[3], kf[2], kf[3]);
                }
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const int t = rt * 16 + g + hf * 8;
                    const float base = DECAY ? 0.0f : F[t] - mt[t];
                    float sum = 0.0f;
#pragma unroll
                    for (int nt = 0; nt < 2; ++nt) {
                        const int key = quarter * 16 + nt * 8 + t4 * 2;
                        auto weight = [&](int k) { return DECAY ? F[t - k] : qscale * expf(base + gx[k]); };
                        const float e0 = key <= t ? p[nt][hf * 2] * weight(key) : 0.0f;
                        const float e1 = key + 1 <= t ? p[nt][hf * 2 + 1] * weight(key + 1) : 0.0f;
                        sum += e0 + e1;
                        split_store(p_hi, p_lo, (size_t)t * CH_P_LD + key, e0, e1);
                    }
                    if (DECAY) continue;
                    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
                    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
                    if (t4 == 0) psum[quarter * CH_L + t] = sum;
                }
            }
            for (int i = tid; i < CH_L * COLS / 2; i += CH_T) {     // values weighted for the state's update, and the ones
                const int r = i / (COLS / 2), x = (i - r * (COLS / 2)) * 2;
                const uint32_t w = *reinterpret_cast<const uint32_t*>(Vc + (size_t)r * LDV + x);
                split_store(wv_hi, wv_lo, (size_t)r * LDV + x, bf16_lo(w) * w_up[r], bf16_hi(w) * w_up[r]);
            }
            if (!DECAY && tid < CH_L) split_store(wv_hi, wv_lo, (size_t)tid * LDV + COLS, w_up[tid], 0.0f);
            asm volatile("bar.sync 1, %0;" ::"n"(CH_T) : "memory");         // (the gate warp has the whole chunk for its work)
            if (OUT) {                                      // O = w_in q^T S + P V, and n.q beside it
                float o[NO][4] = {}, nq[4] = {};
                const uint32_t qa = smem_u32(Qc + (size_t)(rt * 16 + (lm & 1) * 8 + lr) * lay.ld + (lm >> 1) * 8);
                // lanes 0-15 give the rows of the head's tile, lanes 16-31 those of the remainder's
                const uint32_t sb = smem_u32((lm & 2 ? s_lo : s_hi) + (size_t)((lm & 1) * 8 + lr) * LDV);
#pragma unroll 4
                for (int ks = 0; ks < dim / 16; ++ks) {
                    uint32_t qf[4], bf[4];
                    ldsm_x4(qa + ks * 32, qf);
                    if (!DECAY) {
                        ldsm_x4_trans(sb + (uint32_t)(ks * 16 * LDV + COLS) * 2, bf);
                        mma_16816(nq, qf[0], qf[1], qf[2], qf[3], bf[0], bf[1]);
                        mma_16816(nq, qf[0], qf[1], qf[2], qf[3], bf[2], bf[3]);
                    }
#pragma unroll
                    for (int x = 0; x < NO; ++x) {
                        ldsm_x4_trans(sb + (uint32_t)(ks * 16 * LDV + (quarter * NO + x) * 8) * 2, bf);
                        mma_16816(o[x], qf[0], qf[1], qf[2], qf[3], bf[0], bf[1]);
                        mma_16816(o[x], qf[0], qf[1], qf[2], qf[3], bf[2], bf[3]);
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
                for (int ks = 0; ks <= rt; ++ks) {          // keys past the row tile weigh nothing
                    uint32_t ph[4], pl[4];
                    const size_t pat = (size_t)(rt * 16 + (lm & 1) * 8 + lr) * CH_P_LD + ks * 16 + (lm >> 1) * 8;
                    ldsm_x4(smem_u32(p_hi + pat), ph);
                    ldsm_x4(smem_u32(p_lo + pat), pl);
#pragma unroll
                    for (int x = 0; x < NO; ++x) {
                        uint32_t v0, v1;
                        ldsm_x2_trans(smem_u32(Vc + (size_t)(ks * 16 + (lm & 1) * 8 + lr) * LDV + (quarter * NO + x) * 8), v0, v1);
                        mma_16816(o[x], ph[0], ph[1], ph[2], ph[3], v0, v1);
                        mma_16816(o[x], pl[0], pl[1], pl[2], pl[3], v0, v1);
                    }
                }
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const int t = t0 + hf * 8;
                    float inv = 1.0f;
                    if (!DECAY) {
                        float q = __shfl_sync(0xffffffffu, nq[hf * 2], lane & ~3) * (hf ? u1 : u0);       // column 0 of the row
                        if (t < len) {
                            for (int k = 0; k <= rt; ++k) q += psum[k * CH_L + t];
                            inv = 1.0f / (fmaxf(fabsf(q), expf(-mt[t])) + 1e-6f);
                        }
                    }
                    if (t >= len) continue;
                    float* dst = a.out + (size_t)(first + c * CH_L + t) * H * vdim + (size_t)h * vdim;
#pragma unroll
                    for (int x = 0; x < NO; ++x) {
                        const int col = c0 + (quarter * NO + x) * 8 + t4 * 2;
                        if (col < vdim) *reinterpret_cast<float2*>(dst + col) = make_float2(o[x][hf * 2] * inv, o[x][hf * 2 + 1] * inv);
                    }
                }
            }
            if (mine) {                                     // S <- keep S + K^T (weighted values), n likewise
                const float keep = scal[0];
#pragma unroll
                for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
                    for (int e = 0; e < 4; ++e) S[nt][e] *= keep;
#pragma unroll
                for (int e = 0; e < 4; ++e) n[e] *= keep;
                const uint32_t wb = smem_u32((lm & 2 ? wv_lo : wv_hi) + (size_t)((lm & 1) * 8 + lr) * LDV);
#pragma unroll
                for (int ks = 0; ks < CH_L / 16; ++ks) {
                    uint32_t kf[4], bf[4];                  // A = K^T: rows are dimensions, columns tokens
                    ldsm_x4_trans(smem_u32(Kc + (size_t)(ks * 16 + (lm >> 1) * 8 + lr) * lay.ld + r0 + (lm & 1) * 8), kf);
                    if (owns_n) {
                        ldsm_x4_trans(wb + (uint32_t)(ks * 16 * LDV + COLS) * 2, bf);
                        mma_16816(n, kf[0], kf[1], kf[2], kf[3], bf[0], bf[1]);
                        mma_16816(n, kf[0], kf[1], kf[2], kf[3], bf[2], bf[3]);
                    }
#pragma unroll
                    for (int nt = 0; nt < NTS; ++nt) {
                        ldsm_x4_trans(wb + (uint32_t)(ks * 16 * LDV + col0 + nt * 8) * 2, bf);
                        mma_16816(S[nt], kf[0], kf[1], kf[2], kf[3], bf[0], bf[1]);
                        mma_16816(S[nt], kf[0], kf[1], kf[2], kf[3], bf[2], bf[3]);
                    }
                }
            }
        }
        __syncthreads();                                    // before the next chunk rewrites S operands, P and weighted values
    }
    if (MODE == CH_STATES) {
        put_entry(entries + (size_t)(grp + 1) * ENTRY);
        return;
    }
    if (grp != last_grp) return;
    if (mine) {
#pragma unroll
        for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int cc = c0 + col0 + nt * 8 + t4 * 2;
                if (cc < vdim) *reinterpret_cast<float2*>(gs + (size_t)(r0 + g + (e >> 1) * 8) * vdim + cc) = make_float2(S[nt][e], S[nt][e + 1]);
            }
        if (owns_n && t4 == 0)
            for (int sl = 0; sl < nslice; ++sl) {
                gn[(size_t)sl * dim + r0 + g] = n[0];
                gn[(size_t)sl * dim + r0 + g + 8] = n[2];
            }
    } else if (!DECAY && !worker && lane == 0) {
        for (int sl = 0; sl < nslice; ++sl) gm[sl] = m_run;
    }
}

// Columns per CTA and the cut into groups.
struct ChPlan {
    int cols, groups, chunks;
    size_t bytes;
};
ChPlan ch_plan(const scr_mlstm_shape& s, const scr_step& st, int sms) {
    ChPlan p{};
    const int chains = s.heads * st.batch, chunks = scr_ceil_div(st.max_count, CH_L);
    // narrow slices where the wide ones do not fit an SM, or where even all of them leave SMs idle on a short sequence
    p.cols = s.dim > 128 || s.vdim <= 32 || (scr_ceil_div(s.vdim, 32) * chains <= sms && chunks < 8) ? 32 : 64;
    const int ctas = scr_ceil_div(s.vdim, p.cols) * chains;
    p.groups = 1;
    p.chunks = chunks;
    if (chunks >= 8 && 2 * ctas <= sms * 3) {
        // the second pass costs one chunk's update again: cut to about two rounds of CTAs, groups of at least two chunks
        p.groups = std::min(std::max(2, 2 * sms / ctas), chunks / 2);
        p.chunks = scr_ceil_div(chunks, p.groups);
        p.groups = scr_ceil_div(chunks, p.chunks);
    }
    const size_t entry = p.cols == 64 ? ChShape<64, 8>::kEntryFloats : s.dim > 128 ? ChShape<32, 16>::kEntryFloats : ChShape<32, 8>::kEntryFloats;
    p.bytes = p.groups > 1 ? (size_t)ctas * (p.groups + 1) * entry * sizeof(float) : 0;
    return p;
}

template <int COLS, int RTILES, ChMode MODE, bool DECAY>
cudaError_t ch_launch_mode(const MemoryArgs& a, const ChPlan& p, float* ws, cudaStream_t stream) {
    const size_t smem = ChSmem<COLS>::of(a.s.dim).total;
    const cudaError_t e = seq_smem(memory_chunk_kernel<COLS, RTILES, MODE, DECAY>, smem);
    if (e != cudaSuccess) return e;
    return launch_pdl(memory_chunk_kernel<COLS, RTILES, MODE, DECAY>, dim3(scr_ceil_div(a.s.vdim, COLS), a.s.heads, a.st.batch * p.groups), dim3(CH_THREADS), smem, stream, a,
                      ChGroups{ws, p.groups, p.chunks});
}

template <int COLS, int RTILES, bool DECAY>
int32_t ch_launch(scr_ctx* ctx, const MemoryArgs& a, const ChPlan& p, float* ws, cudaStream_t stream) {
    cudaError_t e;
    if (p.groups > 1) {
        e = ch_launch_mode<COLS, RTILES, CH_STATES, DECAY>(a, p, ws, stream);
        if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "memory_chunk states: %s", cudaGetErrorString(e));
        const int32_t rc = scr_check_launch(ctx, "memory_chunk states");
        if (rc) return rc;
        e = ch_launch_mode<COLS, RTILES, CH_OUTPUTS, DECAY>(a, p, ws, stream);
    } else {
        e = ch_launch_mode<COLS, RTILES, CH_WHOLE, DECAY>(a, p, ws, stream);
    }
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "memory_chunk: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "memory_chunk");
}

bool ch_applies(const scr_mlstm_shape& s, const scr_step& st) {
    return st.max_count >= 8 && s.dim % 16 == 0 && s.dim <= 256 && s.vdim % 8 == 0;
}

// The chunks of a step, `workspace` as `ch_plan` wants it.
template <bool DECAY>
int32_t ch_run(scr_ctx* ctx, const MemoryArgs& a, void* workspace, size_t workspace_bytes, cudaStream_t stream) {
    const ChPlan p = ch_plan(a.s, a.st, ctx->sm_count);
    if (p.bytes > workspace_bytes || (p.bytes && !workspace)) return scr_fail(ctx, SCR_E_WORKSPACE, "matrix memory in %d groups needs %zu bytes", p.groups, p.bytes);
    float* ws = (float*)workspace;
    if (a.s.dim > 128) return ch_launch<32, 16, DECAY>(ctx, a, p, ws, stream);
    return p.cols == 64 ? ch_launch<64, 8, DECAY>(ctx, a, p, ws, stream) : ch_launch<32, 8, DECAY>(ctx, a, p, ws, stream);
}

}  // namespace
