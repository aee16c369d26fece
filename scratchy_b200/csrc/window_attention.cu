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
template <typename T> struct Vec<T, 1> {
    static __device__ __forceinline__ void get(const T* p, float (&v)[1]) { v[0] = to_f32(*p); }
    static __device__ __forceinline__ void put(T* p, const float (&v)[1]) { *p = from_f32<T>(v[0]); }
};

// One CTA per ROWS rows.  A thread owns the same channels throughout, keeps their taps and the last projected values in
// registers while it walks the rows, and moves the convolution state of a sequence of one token along itself.
// HIST: taps - 1 where that is small, else -1.
template <typename T, int VEC, int HIST, int ROWS>
__global__ void __launch_bounds__(WP_T) window_prepare_kernel(scr_window_shape s, scr_step st, const T* __restrict__ proj, long long ld,
                                                              const float* __restrict__ conv, const float* __restrict__ norm, T* state,
                                                              T* __restrict__ q, T* __restrict__ cache, float* __restrict__ key_scale, int* status) {
    extern __shared__ float4 wp_smem[];
    float* y = reinterpret_cast<float*>(wp_smem);            // [ROWS][channels]
    __shared__ float red[WP_T / 32][2 * ROWS];
    __shared__ int at_s[ROWS], pos_s[ROWS], count_s[ROWS], slot_s[ROWS];
    __shared__ long long row_s[ROWS];
    pdl_trigger();
    pdl_wait();
    const int r0 = blockIdx.x * ROWS, tid = threadIdx.x;
    const int nq = s.heads * s.dim, C = nq + s.kv_heads * s.dim, hist = HIST >= 0 ? HIST : s.taps - 1;
    if (tid < ROWS) {                                        // at: rows of the portion before this one, -1: no such row
        const int r = r0 + tid, b = r < st.rows ? st.tok_seg[r] : 0;
        const int first = st.segs[b * 4], count = st.segs[b * 4 + 1], slot = st.segs[b * 4 + 3];
        const bool in = r < st.rows && count > 0;
        const bool ok = in && slot >= 0 && slot < st.num_slots && r >= first && r < first + count && first >= 0 && first + count <= st.rows;
        if (in && !ok) atomicCAS(status, 0, SEQ_BAD_SLOT);
        at_s[tid] = ok ? r - first : -1;
        pos_s[tid] = ok ? st.tok_pos[r] : 0;
        count_s[tid] = count;
        slot_s[tid] = slot;
        row_s[tid] = ok ? window_row(s, st.block_table, b, pos_s[tid], status) : -1;
    }
    __syncthreads();
    float sq[ROWS], sk[ROWS];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) sq[i] = sk[i] = 0.0f;
    for (int c = tid * VEC; c < C; c += WP_T * VEC) {
        constexpr int H = HIST >= 0 ? HIST : 1;
        float w[H + 1][VEC], u[H + 1][VEC];                  // u[o]: the token o before this one
        if (HIST >= 0)
#pragma unroll
            for (int o = 0; o <= H; ++o) Vec<float, VEC>::get(conv + (size_t)(hist - o) * C + c, w[o]);
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const int at = at_s[i], r = r0 + i, pos = pos_s[i];
            if (at < 0) continue;
            T* old = state + (size_t)slot_s[i] * hist * C + c;               // oldest first: row hist - d is d tokens before the portion
            auto before = [&](int o, float (&v)[VEC]) {
                if (pos - o < 0) {
#pragma unroll
                    for (int j = 0; j < VEC; ++j) v[j] = 0.0f;
                } else if (o <= at) {
                    Vec<T, VEC>::get(proj + (r - o) * ld + c, v);
                } else {
                    Vec<T, VEC>::get(old + (size_t)(hist - (o - at)) * C, v);
                }
            };
            float acc[VEC], now[VEC];
#pragma unroll
            for (int j = 0; j < VEC; ++j) acc[j] = 0.0f;
            if (HIST >= 0) {
                if (i > 0 && at > 0) {                       // the row before is this sequence's: move along
#pragma unroll
                    for (int o = H; o > 0; --o)
#pragma unroll
                        for (int j = 0; j < VEC; ++j) u[o][j] = u[o - 1][j];
                } else {
#pragma unroll
                    for (int o = H; o > 0; --o) before(o, u[o]);
                }
                Vec<T, VEC>::get(proj + r * ld + c, u[0]);
                if (count_s[i] == 1) {
#pragma unroll
                    for (int o = H; o > 0; --o) Vec<T, VEC>::put(old + (size_t)(hist - o) * C, u[o - 1]);
                }
#pragma unroll
                for (int o = H; o >= 0; --o)
#pragma unroll
                    for (int j = 0; j < VEC; ++j) acc[j] = fmaf(w[o][j], u[o][j], acc[j]);
            } else {
                for (int o = hist; o >= 0; --o) {
                    if (o > 0) before(o, now);
                    else Vec<T, VEC>::get(proj + r * ld + c, now);
                    if (count_s[i] == 1 && o < hist) Vec<T, VEC>::put(old + (size_t)(hist - o - 1) * C, now);
                    Vec<float, VEC>::get(conv + (size_t)(hist - o) * C + c, w[0]);
#pragma unroll
                    for (int j = 0; j < VEC; ++j) acc[j] = fmaf(w[0][j], now[j], acc[j]);
                }
            }
            float ss = 0.0f;
#pragma unroll
            for (int j = 0; j < VEC; ++j) ss = fmaf(acc[j], acc[j], ss);
            Vec<float, VEC>::put(y + (size_t)i * C + c, acc);
            if (c < nq) sq[i] += ss;
            else sk[i] += ss;
        }
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        sq[i] = warp_sum(sq[i]);
        sk[i] = warp_sum(sk[i]);
        if ((tid & 31) == 0) {
            red[tid >> 5][2 * i] = sq[i];
            red[tid >> 5][2 * i + 1] = sk[i];
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        sq[i] = sk[i] = 0.0f;
#pragma unroll
        for (int w = 0; w < WP_T / 32; ++w) {
            sq[i] += red[w][2 * i];
            sk[i] += red[w][2 * i + 1];
        }
        sq[i] = 1.0f / sqrtf(sq[i] / float(nq) + s.eps);
        sk[i] = 1.0f / sqrtf(sk[i] / float(C - nq) + s.eps);
    }
    const int group = s.heads / s.kv_heads;
    for (int c = tid * VEC; c < C; c += WP_T * VEC) {
        float v[VEC], w[VEC], wk[VEC];
        if (c < nq) {
            const int h = c / s.dim;
            Vec<float, VEC>::get(norm + c, w);
            Vec<float, VEC>::get(norm + nq + h / group * s.dim + (c - h * s.dim), wk);
        }
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            if (at_s[i] < 0) continue;
            Vec<float, VEC>::get(y + (size_t)i * C + c, v);
            if (c < nq) {
#pragma unroll
                for (int j = 0; j < VEC; ++j) v[j] = v[j] * sq[i] * w[j] * wk[j];
                Vec<T, VEC>::put(q + (size_t)(r0 + i) * nq + c, v);
            } else if (row_s[i] >= 0) {
                Vec<T, VEC>::put(cache + row_s[i] * (C - nq) + (c - nq), v);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
        if (tid == i && at_s[i] >= 0 && row_s[i] >= 0) key_scale[row_s[i]] = sk[i] * s.scale * 1.4426950408889634f;
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
    const float* bh = bias + (size_t)h * s.n_bias;
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
    const bool many = vec && s.taps <= 4 && st.rows >= 4 * ctx->sm_count && C <= 12 * 1024;
    auto kernel = !vec ? window_prepare_kernel<T, 1, -1, 1> : window_prepare_kernel<T, 8, -1, 1>;
    if (vec && s.taps == 1) kernel = many ? window_prepare_kernel<T, 8, 0, 4> : window_prepare_kernel<T, 8, 0, 1>;
    if (vec && s.taps == 2) kernel = many ? window_prepare_kernel<T, 8, 1, 4> : window_prepare_kernel<T, 8, 1, 1>;
    if (vec && s.taps == 3) kernel = many ? window_prepare_kernel<T, 8, 2, 4> : window_prepare_kernel<T, 8, 2, 1>;
    if (vec && s.taps == 4) kernel = many ? window_prepare_kernel<T, 8, 3, 4> : window_prepare_kernel<T, 8, 3, 1>;
    const int per = many ? 4 : 1;
    const size_t smem = (size_t)per * C * sizeof(float);
    cudaError_t e = seq_smem(kernel, smem);
    if (e == cudaSuccess)
        e = launch_pdl(kernel, dim3(scr_ceil_div(st.rows, per)), dim3(WP_T), smem, stream, s, st, (const T*)proj, (long long)ld, conv, norm, (T*)conv_state, (T*)q,
                       (T*)cache, key_scale, ctx->dev_status);
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
