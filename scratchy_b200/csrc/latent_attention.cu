// Latent attention over the paged cache, in the latent space: the queries already carry W_uk, the values are the latents
// themselves, so every head reads the same cache row [latent | rotated key part].
//
//   latent_attention_plain_kernel   any sizes and both data types, f32 arithmetic
//   latent_attention_mma_kernel     bf16: tensor-core kernel for decoding and short portions (latent_attention_mma.cuh)
// Prompts take the expanded form instead (latent_prefill.cu).
#include "seq_common.cuh"

#include <algorithm>

bool latent_attention_mma_applies(const scr_latent_shape& s);
size_t latent_attention_mma_workspace(const scr_latent_shape& s, const scr_step& st, int sms);
int32_t latent_attention_mma_launch(scr_ctx* ctx, const scr_latent_shape& s, const scr_step& st, const void* q, const void* cache, void* out,
                                    void* workspace, size_t workspace_bytes, cudaStream_t stream);

namespace {

// One CTA per (row, head); its warps take the keys in turn, lanes share a key's dimensions, every warp keeps an online
// softmax state and the states merge in shared memory.
constexpr int LP_WARPS = 8, LP_MAX = 32;                     // up to 32 * 32 latent values

template <typename T>
__global__ void __launch_bounds__(LP_WARPS * 32) latent_attention_plain_kernel(scr_latent_shape s, scr_step st, const T* __restrict__ q,
                                                                               const T* __restrict__ cache, T* __restrict__ out, int* status) {
    extern __shared__ float lp_smem[];
    const int D = s.kv_rank + s.rot_dim;
    float* qs = lp_smem;                                     // [D]
    float* part = qs + D;                                    // [LP_WARPS][kv_rank]
    float* ml = part + LP_WARPS * s.kv_rank;                 // [LP_WARPS][2]
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const T* qp = q + ((size_t)r * s.heads + h) * D;
    for (int i = threadIdx.x; i < D; i += LP_WARPS * 32) qs[i] = to_f32(qp[i]) * s.scale;
    __syncthreads();
    int keys = st.tok_pos[r] + 1;
    if (keys > s.max_blocks * s.block_size) {
        if (threadIdx.x == 0) atomicCAS(status, 0, SEQ_BAD_POSITION);
        keys = s.max_blocks * s.block_size;
    }
    const int* table = st.block_table + (size_t)st.tok_seg[r] * s.max_blocks;
    float m = -INFINITY, l = 0.0f, acc[LP_MAX];
#pragma unroll
    for (int i = 0; i < LP_MAX; ++i) acc[i] = 0.0f;
    for (int t = warp; t < keys; t += LP_WARPS) {
        const int block = table[t / s.block_size];
        if (block < 0 || block >= s.num_blocks) {
            if (lane == 0) atomicCAS(status, 0, SEQ_BAD_BLOCK);
            continue;
        }
        const T* row = cache + ((size_t)block * s.block_size + t % s.block_size) * D;
        float dot = 0.0f;
        for (int i = lane; i < D; i += 32) dot = fmaf(qs[i], to_f32(row[i]), dot);
        dot = warp_sum(dot);
        const float mn = fmaxf(m, dot), keep = expf(m - mn), p = expf(dot - mn);
        l = l * keep + p;
        m = mn;
#pragma unroll
        for (int i = 0; i < LP_MAX; ++i)
            if (i * 32 + lane < s.kv_rank) acc[i] = fmaf(p, to_f32(row[i * 32 + lane]), acc[i] * keep);
    }
#pragma unroll
    for (int i = 0; i < LP_MAX; ++i)
        if (i * 32 + lane < s.kv_rank) part[warp * s.kv_rank + i * 32 + lane] = acc[i];
    if (lane == 0) {
        ml[warp * 2] = m;
        ml[warp * 2 + 1] = l;
    }
    __syncthreads();
    float mt = -INFINITY, lt = 0.0f;
    for (int w = 0; w < LP_WARPS; ++w) mt = fmaxf(mt, ml[w * 2]);
    for (int w = 0; w < LP_WARPS; ++w)
        if (ml[w * 2 + 1] > 0.0f) lt += ml[w * 2 + 1] * expf(ml[w * 2] - mt);
    const float inv = lt > 0.0f ? 1.0f / lt : 0.0f;
    for (int i = threadIdx.x; i < s.kv_rank; i += LP_WARPS * 32) {
        float v = 0.0f;
        for (int w = 0; w < LP_WARPS; ++w)
            if (ml[w * 2 + 1] > 0.0f) v += part[w * s.kv_rank + i] * expf(ml[w * 2] - mt);
        out[((size_t)r * s.heads + h) * s.kv_rank + i] = from_f32<T>(v * inv);
    }
}

template <typename T>
int32_t plain_attention(scr_ctx* ctx, const scr_latent_shape& s, const scr_step& st, const void* q, const void* cache, void* out, cudaStream_t stream) {
    if (s.kv_rank > 32 * LP_MAX) return scr_fail(ctx, SCR_E_UNSUPPORTED, "kv_rank %d", s.kv_rank);
    const size_t smem = (size_t)(s.kv_rank + s.rot_dim + LP_WARPS * s.kv_rank + 2 * LP_WARPS) * sizeof(float);
    cudaError_t e = seq_smem(latent_attention_plain_kernel<T>, smem);
    if (e == cudaSuccess)
        e = launch_pdl(latent_attention_plain_kernel<T>, dim3(st.rows, s.heads), dim3(LP_WARPS * 32), smem, stream, s, st, (const T*)q, (const T*)cache, (T*)out, ctx->dev_status);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "latent_attention: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "latent_attention");
}

}  // namespace

extern "C" int32_t scr_latent_attention_workspace(int32_t dtype, const scr_latent_shape* s, const scr_step* st, size_t* bytes) {
    if (!s || !st || !bytes) return SCR_E_ARG;
    *bytes = dtype == SCR_DTYPE_BF16 && latent_attention_mma_applies(*s) ? latent_attention_mma_workspace(*s, *st, tc_sm_count()) : 0;
    return SCR_OK;
}

extern "C" int32_t scr_latent_attention(scr_ctx* ctx, int32_t dtype, const scr_latent_shape* s, const scr_step* st, const void* q,
                                        const void* cache, void* out, void* workspace, size_t workspace_bytes, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!s || !st || !q || !cache || !out) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (st->rows <= 0 || s->heads <= 0 || s->kv_rank <= 0 || s->block_size <= 0) return scr_fail(ctx, SCR_E_SHAPE, "latent shape");
    if (dtype == SCR_DTYPE_F32) return plain_attention<float>(ctx, *s, *st, q, cache, out, (cudaStream_t)stream);
    if (dtype != SCR_DTYPE_BF16) return scr_fail(ctx, SCR_E_DTYPE, "dtype %d", dtype);
    if (latent_attention_mma_applies(*s))
        return latent_attention_mma_launch(ctx, *s, *st, q, cache, out, workspace, workspace_bytes, (cudaStream_t)stream);
    return plain_attention<bf16>(ctx, *s, *st, q, cache, out, (cudaStream_t)stream);
}
