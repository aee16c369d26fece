// The matrix-memory recurrence (mLSTM) with a stabilised exponential input gate.  Per head, with log gates
//   i = cap tanh((z_i + b_i) / cap),   f = logsigmoid(cap tanh((z_f + b_f) / cap))
// and a running maximum m that starts at 0:
//   m' = max(f + m, i),   S' = e^(f+m-m') S + e^(i-m') k v^T,   n' = e^(f+m-m') n + e^(i-m') k
//   o = S'^T q / (max(|n'.q|, e^(-m')) + 1e-6),   q scaled by dim^(-1/2)
// State and everything about it is f32.
//
//   mlstm_recur_kernel   token by token: decoding, short portions, any sizes, both data types
//   mlstm_chunk.cu       bf16 prompts, 64 tokens at a time on the tensor cores
//   mlstm_finish_kernel  each head's output over its root mean square, the norm's weight and the output gate
#include "seq_common.cuh"
#include "memory.cuh"

#include <algorithm>

bool mlstm_chunk_applies(const scr_mlstm_shape& s, const scr_step& st);
size_t mlstm_chunk_workspace(const scr_mlstm_shape& s, const scr_step& st, int sms);
int32_t mlstm_chunk_launch(scr_ctx* ctx, const MemoryArgs& a, void* workspace, size_t workspace_bytes, cudaStream_t stream);

namespace {

// One CTA per (slice of COLS value columns, head, sequence).  The slice of S stays in shared memory for the whole
// segment; 8 threads with 4 columns each cover a row of it, 32 rows per pass.
constexpr int RC_T = 256, RC_COLS = SCR_MLSTM_SLICE, RC_ROWS = RC_T / 8;

template <typename T>
__global__ void __launch_bounds__(RC_T) mlstm_recur_kernel(MemoryArgs a) {
    extern __shared__ float4 rc_smem[];
    const scr_mlstm_shape& s = a.s;
    const int dim = s.dim, vdim = s.vdim;
    float4* S = rc_smem;                                     // [dim][8] float4
    float* n = reinterpret_cast<float*>(S + (size_t)dim * 8);
    float* qs = n + dim;
    float* ks = qs + dim;
    float4* part = reinterpret_cast<float4*>(ks + dim + (4 - (3 * dim) % 4) % 4);   // [8 warps][8]
    __shared__ float red[2][RC_T / 32];
    pdl_trigger();
    const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * RC_COLS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, cq = tid & 7, row0 = tid >> 3;
    const int* seg = a.st.segs + b * 4;
    const int first = seg[0], count = seg[1], pos0 = seg[2];
    int slot = seg[3];
    pdl_wait();
    if (count <= 0) return;
    if (slot < 0 || slot >= a.st.num_slots || first < 0 || first + count > a.st.rows) {
        if (tid == 0) atomicCAS(a.status, 0, SEQ_BAD_SLOT);
        return;
    }
    const size_t head = (size_t)slot * s.heads + h;
    float* gs = a.state_s + head * dim * vdim;
    // whole float4 columns only: a ragged last column group takes the scalar path
    const int col = c0 + cq * 4, cols_ok = min(4, vdim - col);
    const bool vec = cols_ok == 4 && (vdim & 3) == 0;
    const bool fresh = pos0 == 0;
    const size_t copy = head * mlstm_slices(vdim) + blockIdx.x;          // this slice's own copy of n and m
    float* gn = a.state_n + copy * dim;
    float m = fresh ? 0.0f : a.state_m[copy];
    for (int r = row0; r < dim; r += RC_ROWS) {
        float4 v = make_float4(0, 0, 0, 0);
        if (!fresh) {
            const float* p = gs + (size_t)r * vdim + col;
            if (vec) v = *reinterpret_cast<const float4*>(p);
            else {
                if (cols_ok > 0) v.x = p[0];
                if (cols_ok > 1) v.y = p[1];
                if (cols_ok > 2) v.z = p[2];
                if (cols_ok > 3) v.w = p[3];
            }
        }
        S[r * 8 + cq] = v;
    }
    for (int r = tid; r < dim; r += RC_T) n[r] = fresh ? 0.0f : gn[r];
    const float qscale = 1.0f / sqrtf(float(dim));
    for (int t = 0; t < count; ++t) {
        const int row = first + t;
        const T* p = reinterpret_cast<const T*>(a.proj) + row * a.ld;
        const float gi = mlstm_gate_i(a, row, h), gf = mlstm_gate_f(a, row, h);
        const float mn = fmaxf(gf + m, gi), keep = expf(gf + m - mn), put = expf(gi - mn);
        m = mn;
        float nq = 0.0f;
        for (int r = tid; r < dim; r += RC_T) {
            const float q = to_f32(p[h * dim + r]) * qscale, k = to_f32(p[(s.heads + h) * dim + r]);
            qs[r] = q;
            ks[r] = k;
            const float nn = keep * n[r] + put * k;
            n[r] = nn;
            nq = fmaf(nn, q, nq);
        }
        const T* pv = p + 2 * s.heads * dim + h * vdim + col;
        float4 v = make_float4(0, 0, 0, 0);
        if (cols_ok > 0) v.x = to_f32(pv[0]);
        if (cols_ok > 1) v.y = to_f32(pv[1]);
        if (cols_ok > 2) v.z = to_f32(pv[2]);
        if (cols_ok > 3) v.w = to_f32(pv[3]);
        const float nqt = cta_sum<RC_T>(nq, red[t & 1]);      // (its barrier also publishes qs and ks)
        float4 o = make_float4(0, 0, 0, 0);
        for (int r = row0; r < dim; r += RC_ROWS) {
            float4 e = S[r * 8 + cq];
            const float kp = put * ks[r], q = qs[r];
            e.x = keep * e.x + kp * v.x;
            e.y = keep * e.y + kp * v.y;
            e.z = keep * e.z + kp * v.z;
            e.w = keep * e.w + kp * v.w;
            S[r * 8 + cq] = e;
            o.x = fmaf(e.x, q, o.x);
            o.y = fmaf(e.y, q, o.y);
            o.z = fmaf(e.z, q, o.z);
            o.w = fmaf(e.w, q, o.w);
        }
#pragma unroll
        for (int sh = 8; sh < 32; sh <<= 1) {
            o.x += __shfl_xor_sync(0xffffffffu, o.x, sh);
            o.y += __shfl_xor_sync(0xffffffffu, o.y, sh);
            o.z += __shfl_xor_sync(0xffffffffu, o.z, sh);
            o.w += __shfl_xor_sync(0xffffffffu, o.w, sh);
        }
        if (lane < 8) part[warp * 8 + lane] = o;
        __syncthreads();
        if (tid < RC_COLS && c0 + tid < vdim) {
            float sum = 0.0f;
            for (int w = 0; w < RC_T / 32; ++w) sum += reinterpret_cast<const float*>(part)[w * RC_COLS + tid];
            a.out[(size_t)row * s.heads * vdim + (size_t)h * vdim + c0 + tid] = sum / (fmaxf(fabsf(nqt), expf(-m)) + 1e-6f);
        }
    }
    for (int r = row0; r < dim; r += RC_ROWS) {
        const float4 v = S[r * 8 + cq];
        float* p = gs + (size_t)r * vdim + col;
        if (vec) *reinterpret_cast<float4*>(p) = v;
        else {
            if (cols_ok > 0) p[0] = v.x;
            if (cols_ok > 1) p[1] = v.y;
            if (cols_ok > 2) p[2] = v.z;
            if (cols_ok > 3) p[3] = v.w;
        }
    }
    for (int r = tid; r < dim; r += RC_T) gn[r] = n[r];
    if (tid == 0) a.state_m[copy] = m;
}

constexpr int FIN_T = 128;
template <typename T>
__global__ void __launch_bounds__(FIN_T) mlstm_finish_kernel(scr_mlstm_shape s, const float* __restrict__ out, const float* __restrict__ norm,
                                                             const T* __restrict__ gate, long long ld_gate, T* __restrict__ y) {
    __shared__ float red[FIN_T / 32];
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, r = blockIdx.y;
    const float* o = out + ((size_t)r * s.heads + h) * s.vdim;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < s.vdim; i += FIN_T) ss = fmaf(o[i], o[i], ss);
    const float inv = 1.0f / sqrtf(cta_sum<FIN_T>(ss, red) / float(s.vdim) + s.eps);
    for (int i = threadIdx.x; i < s.vdim; i += FIN_T) {
        const int c = h * s.vdim + i;
        y[(size_t)r * s.heads * s.vdim + c] = from_f32<T>(o[i] * inv * norm[c] * sigmoid_f32(to_f32(gate[r * ld_gate + c])));
    }
}

template <typename T>
int32_t recur_launch(scr_ctx* ctx, const MemoryArgs& a, cudaStream_t stream) {
    const int dim = a.s.dim;
    const size_t smem = (size_t)dim * 8 * 16 + (3 * dim + 4) * sizeof(float) + 8 * 8 * 16;
    if (smem > 220 * 1024) return scr_fail(ctx, SCR_E_UNSUPPORTED, "mlstm dim %d", dim);
    cudaError_t e = seq_smem(mlstm_recur_kernel<T>, smem);
    if (e == cudaSuccess)
        e = launch_pdl(mlstm_recur_kernel<T>, dim3(scr_ceil_div(a.s.vdim, RC_COLS), a.s.heads, a.st.batch), dim3(RC_T), smem, stream, a);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "mlstm_recur: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "mlstm_recur");
}

}  // namespace

extern "C" int32_t scr_mlstm_workspace(int32_t dtype, const scr_mlstm_shape* s, const scr_step* st, size_t* bytes) {
    if (!s || !st || !bytes) return SCR_E_ARG;
    *bytes = dtype == SCR_DTYPE_BF16 && mlstm_chunk_applies(*s, *st) ? mlstm_chunk_workspace(*s, *st, tc_sm_count()) : 0;
    return SCR_OK;
}

extern "C" int32_t scr_mlstm_run(scr_ctx* ctx, int32_t dtype, const scr_mlstm_shape* s, const scr_step* st, const void* proj, int64_t ld,
                                 float* gates, int64_t ld_gates, const float* bias_i, const float* bias_f, float* state_s,
                                 float* state_n, float* state_m, float* out, void* workspace, size_t workspace_bytes,
                                 void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!s || !st || !proj || !gates || !bias_i || !bias_f || !state_s || !state_n || !state_m || !out) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (st->rows <= 0 || st->batch <= 0 || s->heads <= 0 || s->dim <= 0 || s->vdim <= 0) return scr_fail(ctx, SCR_E_SHAPE, "mlstm shape");
    const MemoryArgs a{*s, *st, proj, ld, gates, ld_gates, bias_i, bias_f, state_s, state_n, state_m, out, ctx->dev_status, nullptr};
    if (dtype == SCR_DTYPE_F32) return recur_launch<float>(ctx, a, (cudaStream_t)stream);
    if (dtype != SCR_DTYPE_BF16) return scr_fail(ctx, SCR_E_DTYPE, "dtype %d", dtype);
    if (mlstm_chunk_applies(*s, *st)) return mlstm_chunk_launch(ctx, a, workspace, workspace_bytes, (cudaStream_t)stream);
    return recur_launch<bf16>(ctx, a, (cudaStream_t)stream);
}

extern "C" int32_t scr_mlstm_finish(scr_ctx* ctx, int32_t dtype, const scr_mlstm_shape* s, const float* out, const float* norm,
                                    const void* gate, int64_t ld_gate, int32_t rows, void* y, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!s || !out || !norm || !gate || !y) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (rows <= 0 || rows > 65535) return scr_fail(ctx, SCR_E_SHAPE, "%d rows", rows);
    if (dtype != SCR_DTYPE_F32 && dtype != SCR_DTYPE_BF16) return scr_fail(ctx, SCR_E_DTYPE, "dtype %d", dtype);
    const dim3 grid(s->heads, rows);
    cudaStream_t cs = (cudaStream_t)stream;
    const cudaError_t e = dtype == SCR_DTYPE_F32
        ? launch_pdl(mlstm_finish_kernel<float>, grid, dim3(FIN_T), 0, cs, *s, out, norm, (const float*)gate, (long long)ld_gate, (float*)y)
        : launch_pdl(mlstm_finish_kernel<bf16>, grid, dim3(FIN_T), 0, cs, *s, out, norm, (const bf16*)gate, (long long)ld_gate, (bf16*)y);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "mlstm_finish: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "mlstm_finish");
}
