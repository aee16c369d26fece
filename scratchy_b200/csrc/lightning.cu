// Matrix memory with a constant decay per head (lightning attention): S <- d S + k v^T, o = S^T q, state and sums f32.  A decay close
// to one is applied thousands of times, so it comes as two f32 values.
//
//   lightning_recur_kernel    token by token: decoding, short portions, any sizes, both data types
//   lightning_chunk.cu        bf16 prompts, 64 tokens at a time on the tensor cores
//   lightning_finish_kernel   the concatenated heads over their root mean square, the norm's weight and the output gate
#include "memory.cuh"

bool lightning_chunk_applies(const scr_mlstm_shape& s, const scr_step& st);
size_t lightning_chunk_workspace(const scr_mlstm_shape& s, const scr_step& st, int sms);
int32_t lightning_chunk_launch(scr_ctx* ctx, const MemoryArgs& a, void* workspace, size_t workspace_bytes, cudaStream_t stream);

namespace {

// One CTA per (32 value columns, head, sequence).  The slice of S stays in registers for the whole segment: 8 threads with
// 4 columns each cover a row, a thread has RPT rows, 32 apart.  The state is requested before the wait for the preceding
// kernel (no other kernel of a step touches it).
constexpr int LR_T = 256, LR_COLS = 32, LR_ROWS = LR_T / 8;

template <typename T, int RPT>
__global__ void __launch_bounds__(LR_T) lightning_recur_kernel(MemoryArgs a) {
    __shared__ float4 part[2][LR_T / 32][8];
    pdl_trigger();
    const scr_mlstm_shape& s = a.s;
    const int dim = s.dim, vdim = s.vdim;
    const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * LR_COLS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, row0 = tid >> 3;
    const int* seg = a.st.segs + b * 4;
    const int first = seg[0], count = seg[1], pos0 = seg[2], slot = seg[3];
    const bool ok = count > 0 && slot >= 0 && slot < a.st.num_slots && first >= 0 && first + count <= a.st.rows;
    const int col = c0 + (tid & 7) * 4, cols = min(4, vdim - col);           // this thread's columns that exist
    const bool vec = cols == 4 && (vdim & 3) == 0;
    float* gs = a.state_s + ((size_t)(ok ? slot : 0) * s.heads + h) * dim * vdim + col;
    float4 S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int r = row0 + i * LR_ROWS;
        S[i] = make_float4(0, 0, 0, 0);
        if (ok && pos0 > 0 && r < dim) {
            const float* p = gs + (size_t)r * vdim;
            if (vec) S[i] = *reinterpret_cast<const float4*>(p);
            else {
                if (cols > 0) S[i].x = p[0];
                if (cols > 1) S[i].y = p[1];
                if (cols > 2) S[i].z = p[2];
                if (cols > 3) S[i].w = p[3];
            }
        }
    }
    const float decay = a.powers[(size_t)h * SCR_DECAY_POWERS + 1], rest = a.powers[(size_t)h * SCR_DECAY_POWERS + SCR_DECAY_POWERS - 1];
    pdl_wait();
    if (!ok) {
        if (count > 0 && tid == 0) atomicCAS(a.status, 0, SEQ_BAD_SLOT);
        return;
    }
    float q[RPT], k[RPT], v[4];
    auto fetch = [&](int t) {
        const T* p = reinterpret_cast<const T*>(a.proj) + (first + t) * a.ld;
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const int r = row0 + i * LR_ROWS;
            q[i] = r < dim ? to_f32(p[h * dim + r]) : 0.0f;
            k[i] = r < dim ? to_f32(p[(s.heads + h) * dim + r]) : 0.0f;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] = j < cols ? to_f32(p[2 * s.heads * dim + h * vdim + col + j]) : 0.0f;
    };
    fetch(0);
    for (int t = 0; t < count; ++t) {
        float4 o = make_float4(0, 0, 0, 0);
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            S[i].x = fmaf(decay, S[i].x, fmaf(rest, S[i].x, k[i] * v[0]));
            S[i].y = fmaf(decay, S[i].y, fmaf(rest, S[i].y, k[i] * v[1]));
            S[i].z = fmaf(decay, S[i].z, fmaf(rest, S[i].z, k[i] * v[2]));
            S[i].w = fmaf(decay, S[i].w, fmaf(rest, S[i].w, k[i] * v[3]));
            o.x = fmaf(S[i].x, q[i], o.x);
            o.y = fmaf(S[i].y, q[i], o.y);
            o.z = fmaf(S[i].z, q[i], o.z);
            o.w = fmaf(S[i].w, q[i], o.w);
        }
        if (t + 1 < count) fetch(t + 1);
#pragma unroll
        for (int sh = 8; sh < 32; sh <<= 1) {
            o.x += __shfl_xor_sync(0xffffffffu, o.x, sh);
            o.y += __shfl_xor_sync(0xffffffffu, o.y, sh);
            o.z += __shfl_xor_sync(0xffffffffu, o.z, sh);
            o.w += __shfl_xor_sync(0xffffffffu, o.w, sh);
        }
        if (lane < 8) part[t & 1][warp][lane] = o;
        __syncthreads();                                     // (two buffers: the next token's sums do not wait for this one's readers)
        if (tid < LR_COLS && c0 + tid < vdim) {
            float sum = 0.0f;
#pragma unroll
            for (int w = 0; w < LR_T / 32; ++w) sum += reinterpret_cast<const float*>(part[t & 1][w])[tid];
            a.out[(size_t)(first + t) * s.heads * vdim + (size_t)h * vdim + c0 + tid] = sum;
        }
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int r = row0 + i * LR_ROWS;
        if (r >= dim) continue;
        float* p = gs + (size_t)r * vdim;
        if (vec) *reinterpret_cast<float4*>(p) = S[i];
        else {
            if (cols > 0) p[0] = S[i].x;
            if (cols > 1) p[1] = S[i].y;
            if (cols > 2) p[2] = S[i].z;
            if (cols > 3) p[3] = S[i].w;
        }
    }
}

constexpr int LN_T = 512;
__device__ __forceinline__ void ln_gate(const bf16* p, float (&g)[4]) {
    const uint2 w = *reinterpret_cast<const uint2*>(p);
    g[0] = bf16_lo(w.x); g[1] = bf16_hi(w.x); g[2] = bf16_lo(w.y); g[3] = bf16_hi(w.y);
}
__device__ __forceinline__ void ln_gate(const float* p, float (&g)[4]) {
    const float4 w = *reinterpret_cast<const float4*>(p);
    g[0] = w.x; g[1] = w.y; g[2] = w.z; g[3] = w.w;
}
__device__ __forceinline__ void ln_put(bf16* p, const float (&v)[4]) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3])); }
__device__ __forceinline__ void ln_put(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }

// One CTA per row.  KEEP: runs of 4 values a thread holds in registers between the sum and the product (0: any sizes).
template <typename T, int KEEP>
__global__ void __launch_bounds__(LN_T) lightning_finish_kernel(scr_lightning_shape s, const float* __restrict__ out, const float* __restrict__ norm,
                                                                const T* __restrict__ gate, long long ld_gate, T* __restrict__ y, long long ld_y) {
    __shared__ float red[LN_T / 32];
    pdl_trigger();
    pdl_wait();
    const int n = s.heads * s.vdim, tid = threadIdx.x;
    const size_t r = blockIdx.x;
    const float* o = out + r * n;
    float ss = 0.0f;
    if constexpr (KEEP > 0) {
        constexpr int K = KEEP;
        float v[K][4], w[K][4], g[K][4];
#pragma unroll
        for (int k = 0; k < K; ++k) {
            const int i = (k * LN_T + tid) * 4;
            if (i >= n) continue;
            ln_gate(o + i, v[k]);
            ln_gate(norm + i, w[k]);
            ln_gate(gate + r * ld_gate + i, g[k]);
#pragma unroll
            for (int j = 0; j < 4; ++j) ss = fmaf(v[k][j], v[k][j], ss);
        }
        const float inv = s.out_scale / sqrtf(cta_sum<LN_T>(ss, red) / float(n) + s.eps);
#pragma unroll
        for (int k = 0; k < K; ++k) {
            const int i = (k * LN_T + tid) * 4;
            if (i >= n) continue;
#pragma unroll
            for (int j = 0; j < 4; ++j) v[k][j] = v[k][j] * inv * w[k][j] * sigmoid_f32(g[k][j]);
            ln_put(y + r * ld_y + i, v[k]);
        }
    } else {
        for (int i = tid; i < n; i += LN_T) ss = fmaf(o[i], o[i], ss);
        const float inv = s.out_scale / sqrtf(cta_sum<LN_T>(ss, red) / float(n) + s.eps);
        for (int i = tid; i < n; i += LN_T) y[r * ld_y + i] = from_f32<T>(o[i] * inv * norm[i] * sigmoid_f32(to_f32(gate[r * ld_gate + i])));
    }
}

template <typename T>
int32_t finish(scr_ctx* ctx, const scr_lightning_shape& s, const float* out, const float* norm, const void* gate, int64_t ld_gate, int32_t rows, void* y,
               int64_t ld_y, cudaStream_t stream) {
    const int n = s.heads * s.vdim;
    const bool vec = n % 4 == 0 && ld_gate % 4 == 0 && ld_y % 4 == 0 && scr_aligned16(out) && scr_aligned16(norm) && scr_aligned16(gate) && scr_aligned16(y);
    auto kernel = !vec || n > 16 * LN_T ? lightning_finish_kernel<T, 0> : n > 8 * LN_T ? lightning_finish_kernel<T, 4>
                : n > 4 * LN_T ? lightning_finish_kernel<T, 2> : lightning_finish_kernel<T, 1>;
    const cudaError_t e = launch_pdl(kernel, dim3(rows), dim3(LN_T), 0, stream, s, out, norm, (const T*)gate, (long long)ld_gate, (T*)y, (long long)ld_y);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "lightning_finish: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "lightning_finish");
}

template <typename T, int RPT>
cudaError_t recur(const MemoryArgs& a, cudaStream_t stream) {
    return launch_pdl(lightning_recur_kernel<T, RPT>, dim3(scr_ceil_div(a.s.vdim, LR_COLS), a.s.heads, a.st.batch), dim3(LR_T), 0, stream, a);
}
template <typename T>
int32_t recur_launch(scr_ctx* ctx, const MemoryArgs& a, cudaStream_t stream) {
    const int rows = scr_ceil_div(a.s.dim, LR_ROWS);
    if (rows > 32) return scr_fail(ctx, SCR_E_UNSUPPORTED, "lightning dim %d", a.s.dim);
    const cudaError_t e = rows <= 1 ? recur<T, 1>(a, stream) : rows <= 2 ? recur<T, 2>(a, stream) : rows <= 4 ? recur<T, 4>(a, stream)
                        : rows <= 8 ? recur<T, 8>(a, stream) : recur<T, 32>(a, stream);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "lightning_recur: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "lightning_recur");
}

scr_mlstm_shape memory_shape(const scr_lightning_shape& s) { return scr_mlstm_shape{s.heads, s.dim, s.vdim, 0.0f, s.eps}; }

}  // namespace

extern "C" int32_t scr_lightning_workspace(int32_t dtype, const scr_lightning_shape* s, const scr_step* st, size_t* bytes) {
    if (!s || !st || !bytes) return SCR_E_ARG;
    const scr_mlstm_shape m = memory_shape(*s);
    *bytes = dtype == SCR_DTYPE_BF16 && lightning_chunk_applies(m, *st) ? lightning_chunk_workspace(m, *st, tc_sm_count()) : 0;
    return SCR_OK;
}

extern "C" int32_t scr_lightning_run(scr_ctx* ctx, int32_t dtype, const scr_lightning_shape* s, const scr_step* st, const void* proj, int64_t ld,
                                     const float* powers, float* state, float* out, void* workspace, size_t workspace_bytes, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!s || !st || !proj || !powers || !state || !out) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (st->rows <= 0 || st->batch <= 0 || s->heads <= 0 || s->dim <= 0 || s->vdim <= 0) return scr_fail(ctx, SCR_E_SHAPE, "lightning shape");
    const MemoryArgs a{memory_shape(*s), *st, proj, ld, nullptr, 0, nullptr, nullptr, state, nullptr, nullptr, out, ctx->dev_status, powers};
    if (dtype == SCR_DTYPE_F32) return recur_launch<float>(ctx, a, (cudaStream_t)stream);
    if (dtype != SCR_DTYPE_BF16) return scr_fail(ctx, SCR_E_DTYPE, "dtype %d", dtype);
    if (lightning_chunk_applies(a.s, *st) && ld % 8 == 0 && scr_aligned16(proj))
        return lightning_chunk_launch(ctx, a, workspace, workspace_bytes, (cudaStream_t)stream);
    return recur_launch<bf16>(ctx, a, (cudaStream_t)stream);
}

extern "C" int32_t scr_lightning_finish(scr_ctx* ctx, int32_t dtype, const scr_lightning_shape* s, const float* out, const float* norm,
                                        const void* gate, int64_t ld_gate, int32_t rows, void* y, int64_t ld_y, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!s || !out || !norm || !gate || !y) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (rows <= 0 || s->heads <= 0 || s->vdim <= 0) return scr_fail(ctx, SCR_E_SHAPE, "%d rows", rows);
    if (dtype != SCR_DTYPE_F32 && dtype != SCR_DTYPE_BF16) return scr_fail(ctx, SCR_E_DTYPE, "dtype %d", dtype);
    return dtype == SCR_DTYPE_F32 ? finish<float>(ctx, *s, out, norm, gate, ld_gate, rows, y, ld_y, (cudaStream_t)stream)
                                  : finish<bf16>(ctx, *s, out, norm, gate, ld_gate, rows, y, ld_y, (cudaStream_t)stream);
}
