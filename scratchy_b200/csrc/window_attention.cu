// Sliding-window attention with kept first tokens over a paged cache, whose values are its keys before their norm
// (scr_window_*).  A cache row is the token's convolved key projection, the value of every head; the keys are that row over
// its root mean square times a weight, so the score takes one f32 per token (key_scale) and the queries the weight.
//
//   window_prepare_kernel          short convolution, norm over the whole projection, cache append
//   window_conv_state_kernel       the projected rows that the next portion's convolution reads
//   window_attention_plain_kernel  any sizes and both data types, f32 arithmetic
//   window_attention_mma.cu        bf16: decoding and short portions on mma.sync
//   window_prefill.cu              bf16: prompts on tcgen05
#include "window.cuh"

#include <algorithm>

bool window_mma_applies(const scr_window_shape& s);
int32_t window_mma_launch(scr_ctx* ctx, const scr_window_shape& s, const scr_step& st, const void* q, const void* cache, const float* key_scale,
                          const float* bias, const float* gate, int64_t ld_gate, void* out, int64_t ld_out, cudaStream_t stream);
bool window_prefill_applies(const scr_window_shape& s, const scr_step& st);
int32_t window_prefill_launch(scr_ctx* ctx, const scr_window_shape& s, const scr_step& st, const void* q, const void* cache, const float* key_scale,
                              const float* bias, const float* gate, int64_t ld_gate, void* out, int64_t ld_out, cudaStream_t stream);

namespace {

constexpr int WP_T = 256;

template <typename T, int VEC> struct Vec;
template <> struct Vec<bf16, 8> {
    static __device__ __forceinline__ void get(const bf16* p, float (&v)[8]) {
        const uint4 w = *reinterpret_cast<const uint4*>(p);
        const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            v[2 * i] = bf16_lo(u[i]);
            v[2 * i + 1] = bf16_hi(u[i]);
        }
    }
    static __device__ __forceinline__ void put(bf16* p, const float (&v)[8]) {
        *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
    }
};
template <> struct Vec<float, 8> {
    static __device__ __forceinline__ void get(const float* p, float (&v)[8]) {
#pragma unroll
        for (int i = 0; i < 8; i += 4) {
            const float4 w = *reinterpret_cast<const float4*>(p + i);
            v[i] = w.x; v[i + 1] = w.y; v[i + 2] = w.z; v[i + 3] = w.w;
        }
    }
    static __device__ __forceinline__ void put(float* p, const float (&v)[8]) {
#pragma unroll
        for (int i = 0; i < 8; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    }
};

// What a row of a step is to the convolution: its sequence's portion, slot and cache row.
struct PrepRow {
    long long cache;                                         // -1: none
    int at, pos, count, slot;                                // at: rows of the portion before this one, -1: no such row
};
__device__ __forceinline__ PrepRow prep_row(const scr_window_shape& s, const scr_step& st, int r, int* status) {
    PrepRow p{-1, -1, 0, 0, 0};
    if (r >= st.rows) return p;
    const int b = st.tok_seg[r], first = st.segs[b * 4];
    p.count = st.segs[b * 4 + 1];
    p.slot = st.segs[b * 4 + 3];
    p.pos = st.tok_pos[r];
    if (p.count <= 0) return p;
    if (p.slot < 0 || p.slot >= st.num_slots || r < first || r >= first + p.count || first < 0 || first + p.count > st.rows) {
        atomicCAS(status, 0, SEQ_BAD_SLOT);
        return p;
    }
    p.at = r - first;
    p.cache = window_row(s, st.block_table, b, p.pos, status);
    return p;
}

// One CTA per row, any sizes.  A thread owns the same channels throughout, so that it can move the convolution state of a
// sequence of one token along.
template <typename T>
__global__ void __launch_bounds__(WP_T) window_prepare_any_kernel(scr_window_shape s, scr_step st, const T* __restrict__ proj, long long ld,
                                                                  const float* __restrict__ conv, const float* __restrict__ norm, T* state,
                                                                  T* __restrict__ q, T* __restrict__ cache, float* __restrict__ key_scale, int* status) {
    extern __shared__ float y[];                             // [channels]
    __shared__ float red_q[WP_T / 32], red_k[WP_T / 32];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, tid = threadIdx.x, nq = s.heads * s.dim, C = nq + s.kv_heads * s.dim, hist = s.taps - 1;
    const PrepRow p = prep_row(s, st, r, status);
    if (p.at < 0) return;
    T* old = state + (size_t)p.slot * hist * C;              // oldest first: row hist - d is d tokens before the portion
    float sq = 0.0f, sk = 0.0f;
    for (int c = tid; c < C; c += WP_T) {
        float acc = 0.0f;
        for (int o = hist; o >= 0; --o) {                    // the token o before this one
            T u = from_f32<T>(0.0f);
            if (p.pos - o >= 0) u = o <= p.at ? proj[(r - o) * ld + c] : old[(size_t)(hist - (o - p.at)) * C + c];
            if (p.count == 1 && o < hist) old[(size_t)(hist - o - 1) * C + c] = u;
            acc = fmaf(conv[(size_t)(hist - o) * C + c], to_f32(u), acc);
        }
        y[c] = acc;
        if (c < nq) sq = fmaf(acc, acc, sq);
        else sk = fmaf(acc, acc, sk);
    }
    const float iq = 1.0f / sqrtf(cta_sum<WP_T>(sq, red_q) / float(nq) + s.eps);
    const float ik = 1.0f / sqrtf(cta_sum<WP_T>(sk, red_k) / float(C - nq) + s.eps);
    for (int c = tid; c < C; c += WP_T) {
        if (c < nq) q[(size_t)r * nq + c] = from_f32<T>(y[c] * iq * norm[c]);
        else if (p.cache >= 0) cache[p.cache * (C - nq) + (c - nq)] = from_f32<T>(y[c]);
    }
    if (tid == 0 && p.cache >= 0) key_scale[p.cache] = ik * s.scale * 1.4426950408889634f;
}

// One CTA per ROWS rows, taps <= TAPS: a thread has PER runs of 8 channels, requests the rows and the TAPS - 1 before them at
// once, and keeps everything in registers.  What does not come from the preceding kernel is read before the wait for it.
template <typename T, int TAPS, int PER, int ROWS>
__global__ void __launch_bounds__(512) window_prepare_kernel(scr_window_shape s, scr_step st, const T* __restrict__ proj, long long ld,
                                                             const float* __restrict__ conv, const float* __restrict__ norm, T* state,
                                                             T* __restrict__ q, T* __restrict__ cache, float* __restrict__ key_scale, int* status) {
    constexpr int N = ROWS + TAPS - 1;
    __shared__ float red[16][2 * ROWS];
    __shared__ PrepRow rows[ROWS];
    pdl_trigger();
    const int r0 = blockIdx.x * ROWS, tid = threadIdx.x, nq = s.heads * s.dim, C = nq + s.kv_heads * s.dim, hist = s.taps - 1;
    if (tid < ROWS) rows[tid] = prep_row(s, st, r0 + tid, status);
    __syncthreads();
    float sq[ROWS], sk[ROWS], y[PER][ROWS][8];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) sq[i] = sk[i] = 0.0f;
    if (PER > 1) pdl_wait();
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = (k * blockDim.x + tid) * 8;
        const bool in = c < C;
        float w[TAPS][8];                                    // w[o]: of the token o before
#pragma unroll
        for (int o = 0; o < TAPS; ++o) {
            if (in && o <= hist) {
                Vec<float, 8>::get(conv + (size_t)(hist - o) * C + c, w[o]);
            } else {
#pragma unroll
                for (int j = 0; j < 8; ++j) w[o][j] = 0.0f;
            }
        }
        if (PER == 1) pdl_wait();
        if (!in) continue;
        // what came before the first row: rows of the step, or the state of its sequence
        float u[N][8];
        const PrepRow p0 = rows[0];
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const int o = TAPS - 1 - i;                      // > 0: so many before the first row
            const T* src = nullptr;
            if (o <= 0) src = r0 - o < st.rows ? proj + (r0 - o) * ld + c : nullptr;
            else if (o <= hist && p0.at >= 0 && p0.pos - o >= 0)
                src = o <= p0.at ? proj + (r0 - o) * ld + c : state + ((size_t)p0.slot * hist + (hist - (o - p0.at))) * C + c;
            if (src) Vec<T, 8>::get(src, u[i]);
            else
#pragma unroll
                for (int j = 0; j < 8; ++j) u[i][j] = 0.0f;
        }
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const PrepRow p = rows[i];
            if (p.at < 0) continue;
            float acc[8];
            if (i > 0 && p.at < hist) {                      // a sequence starts within these rows: its own past
#pragma unroll
                for (int o = 1; o < TAPS; ++o)
                    if (o > p.at) {
                        const bool has = o <= hist && p.pos - o >= 0;
                        float v[8];
                        if (has) Vec<T, 8>::get(state + ((size_t)p.slot * hist + (hist - (o - p.at))) * C + c, v);
#pragma unroll
                        for (int j = 0; j < 8; ++j) u[i + TAPS - 1 - o][j] = has ? v[j] : 0.0f;
                    }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[j] = 0.0f;
#pragma unroll
            for (int o = TAPS - 1; o >= 0; --o)
#pragma unroll
                for (int j = 0; j < 8; ++j) acc[j] = fmaf(w[o][j], u[i + TAPS - 1 - o][j], acc[j]);
            float ss = 0.0f;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                ss = fmaf(acc[j], acc[j], ss);
                y[k][i][j] = acc[j];
            }
            if (c < nq) sq[i] += ss;
            else sk[i] += ss;
            if (p.count == 1) {                              // one token: the state moves along (its old rows have been read)
#pragma unroll
                for (int o = TAPS - 1; o > 0; --o)
                    if (o <= hist) Vec<T, 8>::put(state + ((size_t)p.slot * hist + (hist - o)) * C + c, u[i + TAPS - 1 - (o - 1)]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const float a = warp_sum(sq[i]), b = warp_sum(sk[i]);
        if ((tid & 31) == 0) {
            red[tid >> 5][2 * i] = a;
            red[tid >> 5][2 * i + 1] = b;
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        sq[i] = sk[i] = 0.0f;
        for (int w = 0; w < (int)blockDim.x / 32; ++w) {
            sq[i] += red[w][2 * i];
            sk[i] += red[w][2 * i + 1];
        }
        sq[i] = 1.0f / sqrtf(sq[i] / float(nq) + s.eps);
        sk[i] = 1.0f / sqrtf(sk[i] / float(C - nq) + s.eps);
    }
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = (k * blockDim.x + tid) * 8;
        if (c >= C) continue;
        float w[8];
        if (c < nq) Vec<float, 8>::get(norm + c, w);
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const PrepRow p = rows[i];
            if (p.at < 0) continue;
            if (c < nq) {
#pragma unroll
                for (int j = 0; j < 8; ++j) y[k][i][j] *= sq[i] * w[j];
                Vec<T, 8>::put(q + (size_t)(r0 + i) * nq + c, y[k][i]);
            } else if (p.cache >= 0) {
                Vec<T, 8>::put(cache + p.cache * (C - nq) + (c - nq), y[k][i]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
        if (tid == i && rows[i].cache >= 0) key_scale[rows[i].cache] = sk[i] * s.scale * 1.4426950408889634f;
}

// 8 values as they are stored.
template <typename T> struct Raw8;
template <> struct Raw8<bf16> {
    uint4 a;
    __device__ __forceinline__ void load(const bf16* p) { a = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void zero() { a = make_uint4(0, 0, 0, 0); }
    __device__ __forceinline__ float at(int j) const {
        const uint32_t w = j < 2 ? a.x : j < 4 ? a.y : j < 6 ? a.z : a.w;
        return j & 1 ? bf16_hi(w) : bf16_lo(w);
    }
    __device__ __forceinline__ void store(bf16* p) const { *reinterpret_cast<uint4*>(p) = a; }
};
template <> struct Raw8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) {
        a = *reinterpret_cast<const float4*>(p);
        b = *reinterpret_cast<const float4*>(p + 4);
    }
    __device__ __forceinline__ void zero() { a = b = make_float4(0, 0, 0, 0); }
    __device__ __forceinline__ float at(int j) const {
        const float4 v = j < 4 ? a : b;
        return (j & 3) == 0 ? v.x : (j & 3) == 1 ? v.y : (j & 3) == 2 ? v.z : v.w;
    }
    __device__ __forceinline__ void store(float* p) const {
        *reinterpret_cast<float4*>(p) = a;
        *reinterpret_cast<float4*>(p + 4) = b;
    }
};

// Many rows: a CTA walks up to WP_WALK consecutive rows, WP_STEP at a time, with the taps and the last projected values in
// registers; one barrier per step.
constexpr int WP_WALK = 64, WP_STEP = 4;
template <typename T, int TAPS>
__global__ void __launch_bounds__(512) window_prepare_walk_kernel(scr_window_shape s, scr_step st, int per, const T* __restrict__ proj, long long ld,
                                                                  const float* __restrict__ conv, const float* __restrict__ norm, T* state,
                                                                  T* __restrict__ q, T* __restrict__ cache, float* __restrict__ key_scale, int* status) {
    constexpr int PAST = TAPS - 1;
    __shared__ __align__(16) float red[2][16][2][WP_STEP];
    __shared__ PrepRow rows[WP_WALK];
    pdl_trigger();
    const int r0 = blockIdx.x * per, n = min(per, st.rows - r0), tid = threadIdx.x, nq = s.heads * s.dim, C = nq + s.kv_heads * s.dim, hist = s.taps - 1;
    for (int i = tid; i < n; i += blockDim.x) rows[i] = prep_row(s, st, r0 + i, status);
    const int c = tid * 8;
    const bool in = c < C, query = c < nq;
    float w[TAPS][8];                                        // w[o]: of the token o before
#pragma unroll
    for (int o = 0; o < TAPS; ++o) {
#pragma unroll
        for (int j = 0; j < 8; ++j) w[o][j] = 0.0f;
        if (in && o <= hist) Vec<float, 8>::get(conv + (size_t)(hist - o) * C + c, w[o]);
    }
    Raw8<T> u[PAST + WP_STEP];                               // the rows of a step and the PAST before them
#pragma unroll
    for (int i = 0; i < PAST + WP_STEP; ++i) u[i].zero();
    __syncthreads();
    pdl_wait();
#pragma unroll
    for (int o = 1; o < TAPS; ++o)                           // the rows before the first one, where they are of this step
        if (in && o <= hist && o <= rows[0].at) u[PAST - o].load(proj + (r0 - o) * ld + c);
    for (int i0 = 0; i0 < n; i0 += WP_STEP) {
        float y[WP_STEP][8], ss[WP_STEP];
#pragma unroll
        for (int i = 0; i < WP_STEP; ++i)
            if (in && i0 + i < n) u[PAST + i].load(proj + (r0 + i0 + i) * ld + c);
#pragma unroll
        for (int i = 0; i < WP_STEP; ++i) {
            ss[i] = 0.0f;
            if (!in || i0 + i >= n) continue;
            const PrepRow p = rows[i0 + i];
#pragma unroll
            for (int j = 0; j < 8; ++j) y[i][j] = 0.0f;
            if (p.at >= hist) {
#pragma unroll
                for (int o = PAST; o >= 0; --o)
#pragma unroll
                    for (int j = 0; j < 8; ++j) y[i][j] = fmaf(w[o][j], u[PAST + i - o].at(j), y[i][j]);
            } else if (p.at >= 0) {                          // close to its portion's start: what lies before it is in the state
                T* old = state + (size_t)p.slot * hist * C + c;
                Raw8<T> v[TAPS];
#pragma unroll
                for (int o = PAST; o >= 0; --o) {
                    v[o] = u[PAST + i - o];
                    if (o > p.at) {
                        if (o <= hist && p.pos - o >= 0) v[o].load(old + (size_t)(hist - (o - p.at)) * C);
                        else v[o].zero();
                    }
#pragma unroll
                    for (int j = 0; j < 8; ++j) y[i][j] = fmaf(w[o][j], v[o].at(j), y[i][j]);
                }
                if (p.count == 1) {                          // one token: the state moves along
#pragma unroll
                    for (int o = PAST; o > 0; --o)
                        if (o <= hist) v[o - 1].store(old + (size_t)(hist - o) * C);
                }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) ss[i] = fmaf(y[i][j], y[i][j], ss[i]);
        }
#pragma unroll
        for (int i = 0; i < PAST; ++i) u[i] = u[i + WP_STEP];
        float (*sums)[2][WP_STEP] = red[(i0 / WP_STEP) & 1]; // (two sets: the next step's writers need not wait for the readers)
#pragma unroll
        for (int i = 0; i < WP_STEP; ++i) {
            const float a = warp_sum(query ? ss[i] : 0.0f), b = warp_sum(query ? 0.0f : ss[i]);
            if ((tid & 31) == 0) {
                sums[tid >> 5][0][i] = a;
                sums[tid >> 5][1][i] = b;
            }
        }
        __syncthreads();
        float inv[WP_STEP] = {0.0f, 0.0f, 0.0f, 0.0f};
        static_assert(WP_STEP == 4, "a step's sums are one float4");
        for (int k = 0; k < (int)blockDim.x / 32; ++k) {
            const float4 v = *reinterpret_cast<const float4*>(sums[k][query ? 0 : 1]);
            inv[0] += v.x;
            inv[1] += v.y;
            inv[2] += v.z;
            inv[3] += v.w;
        }
        float wn[8];
        if (query) Vec<float, 8>::get(norm + c, wn);
#pragma unroll
        for (int i = 0; i < WP_STEP; ++i) {
            if (!in || i0 + i >= n) continue;
            const PrepRow p = rows[i0 + i];
            if (p.at < 0) continue;
            const float f = 1.0f / sqrtf(inv[i] / float(query ? nq : C - nq) + s.eps);
            if (query) {
#pragma unroll
                for (int j = 0; j < 8; ++j) y[i][j] *= f * wn[j];
                Vec<T, 8>::put(q + (size_t)(r0 + i0 + i) * nq + c, y[i]);
            } else if (p.cache >= 0) {
                Vec<T, 8>::put(cache + p.cache * (C - nq) + (c - nq), y[i]);
                if (c == nq) key_scale[p.cache] = f * s.scale * 1.4426950408889634f;         // (by the thread of the first key channels)
            }
        }
    }
}

// New state row j is the token hist - j before the next portion.  Sources lie behind their destinations, and a thread
// moves a channel's rows in order.
template <typename T>
__global__ void __launch_bounds__(256) window_conv_state_kernel(scr_window_shape s, scr_step st, const T* __restrict__ proj, long long ld, T* state,
                                                                int* status) {
    pdl_trigger();
    pdl_wait();
    const int b = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x, C = (s.heads + s.kv_heads) * s.dim, hist = s.taps - 1;
    const int first = st.segs[b * 4], count = st.segs[b * 4 + 1], pos0 = st.segs[b * 4 + 2], slot = st.segs[b * 4 + 3];
    if (count <= 1 || c >= C) return;                        // (one token: done by the prepare kernel)
    if (slot < 0 || slot >= st.num_slots || first < 0 || first + count > st.rows) {
        atomicCAS(status, 0, SEQ_BAD_SLOT);
        return;
    }
    T* rows = state + (size_t)slot * hist * C + c;
    for (int j = 0; j < hist; ++j) {
        const int i = count - hist + j;                      // row of the portion, negative: before it
        T v = from_f32<T>(0.0f);
        if (i >= 0) v = proj[(first + i) * ld + c];
        else if (pos0 + i >= 0) v = rows[(size_t)(hist + i) * C];
        rows[(size_t)j * C] = v;
    }
}

// One CTA per (row, head); its warps take the visible keys in turn, lanes share a key's dimensions, every warp keeps an
// online softmax state and the states merge in shared memory.
constexpr int WA_WARPS = 8, WA_MAX = 32;                     // up to 32 * 32 dimensions

template <typename T>
__global__ void __launch_bounds__(WA_WARPS * 32) window_attention_plain_kernel(scr_window_shape s, scr_step st, const T* __restrict__ q,
                                                                               const T* __restrict__ cache, const float* __restrict__ key_scale,
                                                                               const float* __restrict__ bias, const float* __restrict__ gate,
                                                                               long long ld_gate, T* __restrict__ out, long long ld_out, int* status) {
    extern __shared__ float wa_smem[];
    float* qs = wa_smem;                                     // [dim]
    float* part = qs + s.dim;                                // [WA_WARPS][dim]
    float* ml = part + WA_WARPS * s.dim;                     // [WA_WARPS][2]
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = h / (s.heads / s.kv_heads);
    const int pos = st.tok_pos[r], seg = st.tok_seg[r];
    const T* qp = q + ((size_t)r * s.heads + h) * s.dim;
    for (int i = threadIdx.x; i < s.dim; i += WA_WARPS * 32) qs[i] = to_f32(qp[i]);
    __syncthreads();
    const int lo = max(0, pos - s.window + 1), kept = min(s.keep_first, lo), keys = kept + pos - lo + 1;
    const float* bh = bias + (size_t)h * (SCR_BIAS_LO + s.n_bias + SCR_BIAS_HI) + SCR_BIAS_LO;
    float m = -INFINITY, l = 0.0f, acc[WA_MAX];
#pragma unroll
    for (int i = 0; i < WA_MAX; ++i) acc[i] = 0.0f;
    for (int t = warp; t < keys; t += WA_WARPS) {
        const int key = t < kept ? t : lo + (t - kept);
        const long long at = window_row(s, st.block_table, seg, key, status);
        if (at < 0) continue;
        const T* row = cache + (at * s.kv_heads + g) * s.dim;
        float dot = 0.0f;
        for (int i = lane; i < s.dim; i += 32) dot = fmaf(qs[i], to_f32(row[i]), dot);
        dot = fmaf(warp_sum(dot), key_scale[at], bh[min(pos - key, s.n_bias - 1)]);
        const float mn = fmaxf(m, dot), keep = exp2f(m - mn), p = exp2f(dot - mn);
        l = l * keep + p;
        m = mn;
#pragma unroll
        for (int i = 0; i < WA_MAX; ++i)
            if (i * 32 + lane < s.dim) acc[i] = fmaf(p, to_f32(row[i * 32 + lane]), acc[i] * keep);
    }
#pragma unroll
    for (int i = 0; i < WA_MAX; ++i)
        if (i * 32 + lane < s.dim) part[warp * s.dim + i * 32 + lane] = acc[i];
    if (lane == 0) {
        ml[warp * 2] = m;
        ml[warp * 2 + 1] = l;
    }
    __syncthreads();
    float mt = -INFINITY, lt = 0.0f;
    for (int w = 0; w < WA_WARPS; ++w) mt = fmaxf(mt, ml[w * 2]);
    for (int w = 0; w < WA_WARPS; ++w)
        if (ml[w * 2 + 1] > 0.0f) lt += ml[w * 2 + 1] * exp2f(ml[w * 2] - mt);
    const float f = lt > 0.0f ? sigmoid_f32(gate[r * ld_gate + h]) * s.out_scale / lt : 0.0f;
    for (int i = threadIdx.x; i < s.dim; i += WA_WARPS * 32) {
        float v = 0.0f;
        for (int w = 0; w < WA_WARPS; ++w)
            if (ml[w * 2 + 1] > 0.0f) v += part[w * s.dim + i] * exp2f(ml[w * 2] - mt);
        out[r * ld_out + (size_t)h * s.dim + i] = from_f32<T>(v * f);
    }
}

int32_t check_shape(scr_ctx* ctx, const scr_window_shape* s, const scr_step* st) {
    if (!s || !st) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (s->heads <= 0 || s->kv_heads <= 0 || s->heads % s->kv_heads || s->dim <= 0 || s->taps <= 0 || s->window <= 0 || s->keep_first < 0 ||
        s->n_bias <= 0 || s->block_size <= 0 || s->num_blocks <= 0 || s->max_blocks <= 0)
        return scr_fail(ctx, SCR_E_SHAPE, "window attention of %d / %d heads, dim %d, taps %d, window %d + %d", s->heads, s->kv_heads, s->dim, s->taps,
                        s->window, s->keep_first);
    if (st->rows <= 0 || st->batch <= 0 || st->max_count <= 0) return scr_fail(ctx, SCR_E_SHAPE, "an empty step");
    return SCR_OK;
}

template <typename T>
int32_t prepare(scr_ctx* ctx, const scr_window_shape& s, const scr_step& st, const void* proj, int64_t ld, const float* conv, const float* norm,
                void* conv_state, void* q, void* cache, float* key_scale, cudaStream_t stream) {
    const int C = (s.heads + s.kv_heads) * s.dim;
    if (C > 50 * 1024) return scr_fail(ctx, SCR_E_UNSUPPORTED, "%d query and key channels", C);
    const bool vec = s.dim % 8 == 0 && ld % 8 == 0 && scr_aligned16(proj) && scr_aligned16(conv) && scr_aligned16(norm) && scr_aligned16(conv_state) &&
                     scr_aligned16(q) && scr_aligned16(cache);
    cudaError_t e;
    if (vec && s.taps <= 4 && C <= 2 * 512 * 8) {
        const bool two = C > 512 * 8;
        const int threads = two ? 512 : scr_ceil_div(C / 8, 32) * 32;
        if (!two && st.rows >= 2 * ctx->sm_count) {
            const int per = std::min(WP_WALK, std::max(WP_STEP, scr_ceil_div(scr_ceil_div(st.rows, ctx->sm_count), WP_STEP) * WP_STEP));
            e = launch_pdl(window_prepare_walk_kernel<T, 4>, dim3(scr_ceil_div(st.rows, per)), dim3(threads), 0, stream, s, st, per, (const T*)proj, (long long)ld,
                           conv, norm, (T*)conv_state, (T*)q, (T*)cache, key_scale, ctx->dev_status);
        } else {
            auto kernel = !two ? window_prepare_kernel<T, 4, 1, 1> : st.rows >= 2 * ctx->sm_count ? window_prepare_kernel<T, 4, 2, 2> : window_prepare_kernel<T, 4, 2, 1>;
            const int per = two && st.rows >= 2 * ctx->sm_count ? 2 : 1;
            e = launch_pdl(kernel, dim3(scr_ceil_div(st.rows, per)), dim3(threads), 0, stream, s, st, (const T*)proj, (long long)ld, conv, norm, (T*)conv_state, (T*)q,
                           (T*)cache, key_scale, ctx->dev_status);
        }
    } else {
        const size_t smem = (size_t)C * sizeof(float);
        e = seq_smem(window_prepare_any_kernel<T>, smem);
        if (e == cudaSuccess)
            e = launch_pdl(window_prepare_any_kernel<T>, dim3(st.rows), dim3(WP_T), smem, stream, s, st, (const T*)proj, (long long)ld, conv, norm, (T*)conv_state,
                           (T*)q, (T*)cache, key_scale, ctx->dev_status);
    }
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "window_prepare: %s", cudaGetErrorString(e));
    const int32_t rc = scr_check_launch(ctx, "window_prepare");
    if (rc || st.max_count == 1 || s.taps == 1) return rc;
    e = launch_pdl(window_conv_state_kernel<T>, dim3(scr_ceil_div(C, 256), st.batch), dim3(256), 0, stream, s, st, (const T*)proj, (long long)ld,
                   (T*)conv_state, ctx->dev_status);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "window_conv_state: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "window_conv_state");
}

template <typename T>
int32_t plain_attention(scr_ctx* ctx, const scr_window_shape& s, const scr_step& st, const void* q, const void* cache, const float* key_scale,
                        const float* bias, const float* gate, int64_t ld_gate, void* out, int64_t ld_out, cudaStream_t stream) {
    if (s.dim > 32 * WA_MAX) return scr_fail(ctx, SCR_E_UNSUPPORTED, "dim %d", s.dim);
    const size_t smem = (size_t)(s.dim + WA_WARPS * s.dim + 2 * WA_WARPS) * sizeof(float);
    cudaError_t e = seq_smem(window_attention_plain_kernel<T>, smem);
    if (e == cudaSuccess)
        e = launch_pdl(window_attention_plain_kernel<T>, dim3(st.rows, s.heads), dim3(WA_WARPS * 32), smem, stream, s, st, (const T*)q, (const T*)cache,
                       key_scale, bias, gate, (long long)ld_gate, (T*)out, (long long)ld_out, ctx->dev_status);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "window_attention: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "window_attention");
}

}  // namespace

extern "C" int32_t scr_window_prepare(scr_ctx* ctx, int32_t dtype, const scr_window_shape* s, const scr_step* st, const void* proj, int64_t ld,
                                      const float* conv, const float* norm, void* conv_state, void* q, void* cache, float* key_scale, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    const int32_t rc = check_shape(ctx, s, st);
    if (rc) return rc;
    if (!proj || !conv || !norm || !conv_state || !q || !cache || !key_scale) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (dtype == SCR_DTYPE_F32) return prepare<float>(ctx, *s, *st, proj, ld, conv, norm, conv_state, q, cache, key_scale, (cudaStream_t)stream);
    if (dtype != SCR_DTYPE_BF16) return scr_fail(ctx, SCR_E_DTYPE, "dtype %d", dtype);
    return prepare<bf16>(ctx, *s, *st, proj, ld, conv, norm, conv_state, q, cache, key_scale, (cudaStream_t)stream);
}

extern "C" int32_t scr_window_attention(scr_ctx* ctx, int32_t dtype, const scr_window_shape* s, const scr_step* st, const void* q, const void* cache,
                                        const float* key_scale, const float* bias, const float* gate, int64_t ld_gate, void* out, int64_t ld_out,
                                        void* stream) {
    SCR_REQUIRE_CTX(ctx);
    const int32_t rc = check_shape(ctx, s, st);
    if (rc) return rc;
    if (!q || !cache || !key_scale || !bias || !gate || !out) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    cudaStream_t cs = (cudaStream_t)stream;
    if (dtype == SCR_DTYPE_F32) return plain_attention<float>(ctx, *s, *st, q, cache, key_scale, bias, gate, ld_gate, out, ld_out, cs);
    if (dtype != SCR_DTYPE_BF16) return scr_fail(ctx, SCR_E_DTYPE, "dtype %d", dtype);
    const bool aligned = scr_aligned16(q) && scr_aligned16(cache) && scr_aligned16(key_scale) && scr_aligned16(out) && ld_out % 8 == 0;
    if (aligned && window_prefill_applies(*s, *st)) return window_prefill_launch(ctx, *s, *st, q, cache, key_scale, bias, gate, ld_gate, out, ld_out, cs);
    if (aligned && window_mma_applies(*s)) return window_mma_launch(ctx, *s, *st, q, cache, key_scale, bias, gate, ld_gate, out, ld_out, cs);
    return plain_attention<bf16>(ctx, *s, *st, q, cache, key_scale, bias, gate, ld_gate, out, ld_out, cs);
}
