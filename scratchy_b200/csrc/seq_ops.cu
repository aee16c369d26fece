// The row operators of the sequence models: embedding, the norms between sublayers on the f32 residual stream, the
// latent projections' norms with rotation and cache append, query rotation, cache gather and greedy argmax.  Byte movers
// bounded by HBM or launch latency.
#include "seq_common.cuh"

namespace {

// ------------------------------------------------------------------------------- embedding
template <typename T>
__global__ void seq_embed_kernel(const int* __restrict__ ids, const T* __restrict__ table, int vocab, int width, float* __restrict__ x,
                                 T* __restrict__ raw, long long ld_raw, int* status) {
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, id = ids[r];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0) atomicCAS(status, 0, SEQ_BAD_TOKEN_ID);
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const T v = ok ? table[(size_t)id * width + i] : from_f32<T>(0.0f);
        x[(size_t)r * width + i] = to_f32(v);
        if (raw) raw[r * ld_raw + i] = v;
    }
}

// ------------------------------------------------------------------------------- norms between sublayers
constexpr int NORM_T = 256;

__device__ __forceinline__ void put_vec(float* dst, const float (&v)[4]) { *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void put_vec(bf16* dst, const float (&v)[4]) { *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3])); }
__device__ __forceinline__ void put_vec(float* dst, const float (&v)[1]) { *dst = v[0]; }
__device__ __forceinline__ void put_vec(bf16* dst, const float (&v)[1]) { *dst = __float2bfloat16_rn(v[0]); }
__device__ __forceinline__ void get_vec(const float* src, float (&v)[4]) {
    const float4 q = *reinterpret_cast<const float4*>(src);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
}
__device__ __forceinline__ void get_vec(const float* src, float (&v)[1]) { v[0] = *src; }

// One CTA per row.  The row lives in shared memory between the passes.
template <typename T, int VEC>
__global__ void __launch_bounds__(NORM_T) seq_norm_kernel(scr_seq_norm_args a, int* status) {
    extern __shared__ float4 norm_row[];
    float* row = reinterpret_cast<float*>(norm_row);
    __shared__ float red_a[NORM_T / 32], red_b[NORM_T / 32];
    pdl_trigger();
    pdl_wait();
    const int W = a.width, r = blockIdx.x;
    int src = r;
    if (a.row_index) {
        src = a.row_index[r];
        if (src < 0 || src >= a.x_rows) {
            if (threadIdx.x == 0) atomicCAS(status, 0, SEQ_BAD_POSITION);
            src = 0;
        }
    }
    float* x = a.x + (size_t)src * W;
    float sum = 0.0f;
    if (a.delta) {
        const float* d = a.delta + (size_t)r * W;
        float ss = 0.0f;
        for (int i = threadIdx.x * VEC; i < W; i += NORM_T * VEC) {
            float v[VEC];
            get_vec(d + i, v);
            put_vec(row + i, v);
#pragma unroll
            for (int j = 0; j < VEC; ++j) ss = fmaf(v[j], v[j], ss);
        }
        float inv = 0.0f;
        if (a.w_delta) inv = 1.0f / sqrtf(cta_sum<NORM_T>(ss, red_a) / float(W) + a.eps);
        for (int i = threadIdx.x * VEC; i < W; i += NORM_T * VEC) {       // each thread reads back its own elements
            float v[VEC], o[VEC], w[VEC];
            get_vec(row + i, v);
            if (a.w_delta) {
                get_vec(x + i, o);
                get_vec(a.w_delta + i, w);
#pragma unroll
                for (int j = 0; j < VEC; ++j) o[j] += v[j] * inv * (1.0f + w[j]);
            } else {
#pragma unroll
                for (int j = 0; j < VEC; ++j) w[j] = 0.0f;
                if (a.bias) get_vec(a.bias + i, w);
#pragma unroll
                for (int j = 0; j < VEC; ++j) o[j] = v[j] + w[j];
            }
            put_vec(x + i, o);
            put_vec(row + i, o);
#pragma unroll
            for (int j = 0; j < VEC; ++j) sum = fmaf(o[j], o[j], sum);
        }
    } else {
        for (int i = threadIdx.x * VEC; i < W; i += NORM_T * VEC) {
            float v[VEC];
            get_vec(x + i, v);
            put_vec(row + i, v);
#pragma unroll
            for (int j = 0; j < VEC; ++j) sum = fmaf(v[j], v[j], sum);
        }
    }
    if (!a.out) return;
    T* out = reinterpret_cast<T*>(a.out) + r * a.ld_out;
    float inv = 1.0f;
    if (a.w_out && !a.b_out) inv = 1.0f / sqrtf(cta_sum<NORM_T>(sum, red_b) / float(W) + a.eps);
    for (int i = threadIdx.x * VEC; i < W; i += NORM_T * VEC) {
        float v[VEC], w[VEC];
        get_vec(row + i, v);
        if (a.b_out) {
            float b[VEC];
            get_vec(a.w_out + i, w);
            get_vec(a.b_out + i, b);
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] = fmaf(tanhf(a.alpha * v[j]), w[j], b[j]);
        } else if (a.w_out) {
            get_vec(a.w_out + i, w);
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] = v[j] * inv * (1.0f + w[j]);
        }
        put_vec(out + i, v);
    }
}

// ------------------------------------------------------------------------------- greedy argmax
constexpr int AMAX_T = 1024;
__device__ __forceinline__ void amax_take(float v, int i, float& best, int& best_i) {
    if (v > best || (v == best && i < best_i)) {
        best = v;
        best_i = i;
    }
}
__global__ void __launch_bounds__(AMAX_T) seq_argmax_kernel(const float* __restrict__ logits, long long ld, int width, int* __restrict__ out) {
    __shared__ float sb[AMAX_T / 32];
    __shared__ int si[AMAX_T / 32];
    pdl_trigger();
    pdl_wait();
    const float* row = logits + blockIdx.x * ld;
    float best = -INFINITY;
    int best_i = 0x7FFFFFFF;
    for (int i = threadIdx.x; i < width; i += AMAX_T) amax_take(row[i], i, best, best_i);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, best_i, o);
        amax_take(ob, oi, best, best_i);
    }
    if ((threadIdx.x & 31) == 0) {
        sb[threadIdx.x >> 5] = best;
        si[threadIdx.x >> 5] = best_i;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < AMAX_T / 32; ++w) amax_take(sb[w], si[w], best, best_i);
        out[blockIdx.x] = best_i == 0x7FFFFFFF ? 0 : best_i;
    }
}

// ------------------------------------------------------------------------------- latent projections -> query latent, cache row
// Where the row of (sequence seg, position pos) lives in a paged cache; -1 (and a status code) outside it.
__device__ __forceinline__ long long cache_row(const scr_latent_shape& s, const int* block_table, int seg, int pos, int* status) {
    const int b = pos / s.block_size;
    if (pos < 0 || b >= s.max_blocks) {
        atomicCAS(status, 0, SEQ_BAD_POSITION);
        return -1;
    }
    const int block = block_table[(size_t)seg * s.max_blocks + b];
    if (block < 0 || block >= s.num_blocks) {
        atomicCAS(status, 0, SEQ_BAD_BLOCK);
        return -1;
    }
    return (long long)block * s.block_size + (pos - b * s.block_size);
}

// The interleaved rotation of value i of a vector whose first `dims` values rotate: pair (2j, 2j + 1).
template <typename F>
__device__ __forceinline__ float rotated(F at, int i, int dims, const float* cs, const float* sn) {
    if (i >= dims) return at(i);
    const int j = i >> 1;
    return (i & 1) ? at(i) * cs[j] + at(i - 1) * sn[j] : at(i) * cs[j] - at(i + 1) * sn[j];
}

constexpr int PREP_T = 128;
template <typename T>
__global__ void __launch_bounds__(PREP_T) latent_prepare_kernel(scr_latent_shape s, scr_step st, const float* __restrict__ d, long long ld_d,
                                                               const float* __restrict__ wq, const float* __restrict__ wkv,
                                                               const float* __restrict__ cos_table, const float* __restrict__ sin_table,
                                                               T* __restrict__ c_q, T* __restrict__ cache, int* status) {
    __shared__ float red_a[PREP_T / 32], red_b[PREP_T / 32];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, tid = threadIdx.x;
    const float *dq = d + r * ld_d, *dc = dq + s.q_rank, *dr = dc + s.kv_rank;
    float sq = 0.0f, sc = 0.0f;
    for (int i = tid; i < s.q_rank; i += PREP_T) sq = fmaf(dq[i], dq[i], sq);
    for (int i = tid; i < s.kv_rank; i += PREP_T) sc = fmaf(dc[i], dc[i], sc);
    const float iq = 1.0f / sqrtf(cta_sum<PREP_T>(sq, red_a) / float(s.q_rank) + s.eps);
    const float ic = 1.0f / sqrtf(cta_sum<PREP_T>(sc, red_b) / float(s.kv_rank) + s.eps);
    for (int i = tid; i < s.q_rank; i += PREP_T) c_q[(size_t)r * s.q_rank + i] = from_f32<T>(dq[i] * iq * wq[i]);
    const int pos = st.tok_pos[r];
    const long long row = cache_row(s, st.block_table, st.tok_seg[r], pos, status);
    if (row < 0) return;
    if (pos >= s.max_pos) {
        if (tid == 0) atomicCAS(status, 0, SEQ_BAD_POSITION);
        return;
    }
    T* dst = cache + row * (s.kv_rank + s.rot_dim);
    for (int i = tid; i < s.kv_rank; i += PREP_T) dst[i] = from_f32<T>(dc[i] * ic * wkv[i]);
    const float *cs = cos_table + (size_t)pos * (s.rot_dims / 2), *sn = sin_table + (size_t)pos * (s.rot_dims / 2);
    for (int i = tid; i < s.rot_dim; i += PREP_T)
        dst[s.kv_rank + i] = from_f32<T>(rotated([&](int j) { return dr[j]; }, i, s.rot_dims, cs, sn));
}

template <typename T>
__global__ void __launch_bounds__(256) latent_queries_kernel(scr_latent_shape s, scr_step st, const float* __restrict__ q,
                                                             const float* __restrict__ cos_table, const float* __restrict__ sin_table,
                                                             T* __restrict__ q_plain, long long ld_plain, long long head_plain,
                                                             T* __restrict__ q_rot, long long ld_rot, long long head_rot, int* status) {
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, per = s.dim + s.rot_dim;
    int pos = st.tok_pos[r];
    if (pos < 0 || pos >= s.max_pos) {
        if (threadIdx.x == 0) atomicCAS(status, 0, SEQ_BAD_POSITION);
        pos = 0;
    }
    const float *cs = cos_table + (size_t)pos * (s.rot_dims / 2), *sn = sin_table + (size_t)pos * (s.rot_dims / 2);
    for (int i = threadIdx.x; i < s.heads * per; i += 256) {
        const int h = i / per, e = i - h * per;
        const float* src = q + (size_t)r * s.heads * per + (size_t)h * per;
        if (e < s.dim) q_plain[r * ld_plain + h * head_plain + e] = from_f32<T>(src[e]);
        else q_rot[r * ld_rot + h * head_rot + e - s.dim] = from_f32<T>(rotated([&](int j) { return src[s.dim + j]; }, e - s.dim, s.rot_dims, cs, sn));
    }
}

__global__ void __launch_bounds__(128) latent_gather_kernel(scr_latent_shape s, const int* __restrict__ table, const bf16* __restrict__ cache,
                                                            bf16* __restrict__ c, bf16* __restrict__ r, int* status) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const long long row = cache_row(s, table, 0, t, status);
    if (row < 0) return;
    const bf16* src = cache + row * (s.kv_rank + s.rot_dim);
    for (int i = threadIdx.x; i < s.kv_rank; i += 128) c[(size_t)t * s.kv_rank + i] = src[i];
    for (int i = threadIdx.x; i < s.rot_dim; i += 128) r[(size_t)t * s.rot_dim + i] = src[s.kv_rank + i];
}

}  // namespace

#define SEQ_LAUNCH(what, call)                                                                                     \
    do {                                                                                                           \
        const cudaError_t e_ = (call);                                                                             \
        if (e_ != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "%s: %s", what, cudaGetErrorString(e_));           \
        return scr_check_launch(ctx, what);                                                                        \
    } while (0)
#define SEQ_DTYPE(dtype)                                                                                           \
    if ((dtype) != SCR_DTYPE_F32 && (dtype) != SCR_DTYPE_BF16) return scr_fail(ctx, SCR_E_DTYPE, "dtype %d", dtype)

extern "C" int32_t scr_seq_embed(scr_ctx* ctx, int32_t dtype, const int32_t* ids, int32_t rows, const void* table, int32_t vocab,
                                 int32_t width, float* x, void* raw, int64_t ld_raw, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    SEQ_DTYPE(dtype);
    if (!ids || !table || !x) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (rows <= 0 || vocab <= 0 || width <= 0) return scr_fail(ctx, SCR_E_SHAPE, "empty embedding");
    cudaStream_t st = (cudaStream_t)stream;
    if (dtype == SCR_DTYPE_F32)
        SEQ_LAUNCH("seq_embed", launch_pdl(seq_embed_kernel<float>, dim3(rows), dim3(256), 0, st, ids, (const float*)table, vocab, width, x, (float*)raw, (long long)ld_raw, ctx->dev_status));
    SEQ_LAUNCH("seq_embed", launch_pdl(seq_embed_kernel<bf16>, dim3(rows), dim3(256), 0, st, ids, (const bf16*)table, vocab, width, x, (bf16*)raw, (long long)ld_raw, ctx->dev_status));
}

extern "C" int32_t scr_seq_norm(scr_ctx* ctx, int32_t dtype, const scr_seq_norm_args* ap, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    SEQ_DTYPE(dtype);
    if (!ap || !ap->x || (ap->row_index && ap->delta) || (ap->b_out && !ap->w_out)) return scr_fail(ctx, SCR_E_ARG, "null pointer, or a row index together with a delta");
    const scr_seq_norm_args& a = *ap;
    if (a.rows <= 0 || a.width <= 0) return scr_fail(ctx, SCR_E_SHAPE, "empty norm");
    const size_t smem = (size_t)a.width * sizeof(float);
    if (smem > 200 * 1024) return scr_fail(ctx, SCR_E_UNSUPPORTED, "width %d", a.width);
    const bool vec = a.width % 4 == 0 && a.ld_out % 4 == 0 && scr_aligned16(a.x) && scr_aligned16(a.delta) && scr_aligned16(a.w_delta) &&
                     scr_aligned16(a.bias) && scr_aligned16(a.w_out) && scr_aligned16(a.b_out) && scr_aligned16(a.out);
    auto kernel = dtype == SCR_DTYPE_F32 ? (vec ? seq_norm_kernel<float, 4> : seq_norm_kernel<float, 1>) : (vec ? seq_norm_kernel<bf16, 4> : seq_norm_kernel<bf16, 1>);
    cudaError_t e = seq_smem(kernel, smem);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "seq_norm: %s", cudaGetErrorString(e));
    SEQ_LAUNCH("seq_norm", launch_pdl(kernel, dim3(a.rows), dim3(NORM_T), smem, (cudaStream_t)stream, a, ctx->dev_status));
}

extern "C" int32_t scr_seq_argmax(scr_ctx* ctx, const float* logits, int64_t ld, int32_t rows, int32_t width, int32_t* out, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!logits || !out) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (rows <= 0 || width <= 0) return scr_fail(ctx, SCR_E_SHAPE, "empty argmax");
    SEQ_LAUNCH("seq_argmax", launch_pdl(seq_argmax_kernel, dim3(rows), dim3(AMAX_T), 0, (cudaStream_t)stream, logits, (long long)ld, width, out));
}

extern "C" int32_t scr_latent_prepare(scr_ctx* ctx, int32_t dtype, const scr_latent_shape* s, const scr_step* st, const float* d, int64_t ld_d,
                                      const float* wq_norm, const float* wkv_norm, const float* cos_table, const float* sin_table,
                                      void* c_q, void* cache, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    SEQ_DTYPE(dtype);
    if (!s || !st || !d || !wq_norm || !wkv_norm || !c_q || !cache) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (st->rows <= 0 || s->rot_dims % 2 || s->rot_dims > s->rot_dim || s->block_size <= 0) return scr_fail(ctx, SCR_E_SHAPE, "latent shape");
    cudaStream_t cs = (cudaStream_t)stream;
    if (dtype == SCR_DTYPE_F32)
        SEQ_LAUNCH("latent_prepare", launch_pdl(latent_prepare_kernel<float>, dim3(st->rows), dim3(PREP_T), 0, cs, *s, *st, d, (long long)ld_d, wq_norm, wkv_norm, cos_table, sin_table, (float*)c_q, (float*)cache, ctx->dev_status));
    SEQ_LAUNCH("latent_prepare", launch_pdl(latent_prepare_kernel<bf16>, dim3(st->rows), dim3(PREP_T), 0, cs, *s, *st, d, (long long)ld_d, wq_norm, wkv_norm, cos_table, sin_table, (bf16*)c_q, (bf16*)cache, ctx->dev_status));
}

extern "C" int32_t scr_latent_queries(scr_ctx* ctx, int32_t dtype, const scr_latent_shape* s, const scr_step* st, const float* q,
                                      const float* cos_table, const float* sin_table, void* q_plain, int64_t ld_plain, int64_t head_plain,
                                      void* q_rot, int64_t ld_rot, int64_t head_rot, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    SEQ_DTYPE(dtype);
    if (!s || !st || !q || !q_plain || !q_rot) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (st->rows <= 0 || s->rot_dims % 2 || s->rot_dims > s->rot_dim) return scr_fail(ctx, SCR_E_SHAPE, "latent shape");
    cudaStream_t cs = (cudaStream_t)stream;
    if (dtype == SCR_DTYPE_F32)
        SEQ_LAUNCH("latent_queries", launch_pdl(latent_queries_kernel<float>, dim3(st->rows), dim3(256), 0, cs, *s, *st, q, cos_table, sin_table, (float*)q_plain, (long long)ld_plain, (long long)head_plain, (float*)q_rot, (long long)ld_rot, (long long)head_rot, ctx->dev_status));
    SEQ_LAUNCH("latent_queries", launch_pdl(latent_queries_kernel<bf16>, dim3(st->rows), dim3(256), 0, cs, *s, *st, q, cos_table, sin_table, (bf16*)q_plain, (long long)ld_plain, (long long)head_plain, (bf16*)q_rot, (long long)ld_rot, (long long)head_rot, ctx->dev_status));
}

extern "C" int32_t scr_latent_gather(scr_ctx* ctx, const scr_latent_shape* s, const int32_t* block_table_row, int32_t kv, const void* cache,
                                     void* c, void* r, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!s || !block_table_row || !cache || !c || !r) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (kv <= 0) return scr_fail(ctx, SCR_E_SHAPE, "empty gather");
    SEQ_LAUNCH("latent_gather", launch_pdl(latent_gather_kernel, dim3(kv), dim3(128), 0, (cudaStream_t)stream, *s, block_table_row, (const bf16*)cache, (bf16*)c, (bf16*)r, ctx->dev_status));
}
