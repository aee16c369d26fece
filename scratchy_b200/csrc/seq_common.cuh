// Shared helpers of the sequence-model kernels (include/scratchy_models.h).
#pragma once

#include "tc_common.cuh"
#include "../../include/scratchy_models.h"

// Codes of device-side argument checks (`scr_device_status` reports SCR_E_ARG; the access is skipped).
constexpr int SEQ_BAD_TOKEN_ID = 0x0E000001;
constexpr int SEQ_BAD_SLOT = 0x0E000002;
constexpr int SEQ_BAD_BLOCK = 0x0E000003;
constexpr int SEQ_BAD_POSITION = 0x0E000004;

typedef __nv_bfloat16 bf16;

// Programmatic dependent launch: a kernel lets its successor start its prologue at once and waits for its
// predecessors' results before it touches anything a kernel of the step writes.
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

template <typename... KArgs, typename... Args>
static inline cudaError_t launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

// Raises a kernel's dynamic shared memory limit where a launch needs more than the default 48 KB.
template <typename K>
static inline cudaError_t seq_smem(K kernel, size_t bytes) {
    return bytes > 48 * 1024 ? cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) : cudaSuccess;
}

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
    const __nv_bfloat162 p = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&p);
}
__device__ __forceinline__ float bf16_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t w) { return __uint_as_float(w & 0xFFFF0000u); }

__device__ __forceinline__ float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }

// a sigmoid(alpha a) (b + 1) with a = min(gate, limit), b = clamp(up, -limit, limit)
__device__ __forceinline__ float clamped_glu(float gate, float up, float limit, float alpha) {
    const float a = fminf(gate, limit), b = fminf(fmaxf(up, -limit), limit);
    return a * sigmoid_f32(alpha * a) * (b + 1.0f);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Sum over a CTA of THREADS threads; every thread gets it.  `red`: THREADS / 32 floats, reusable after the next barrier.
template <int THREADS>
__device__ __forceinline__ float cta_sum(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) t += red[w];
    return t;
}

// D(16x8,f32) += A(16x16,bf16) * B(16x8,bf16)
__device__ __forceinline__ void mma_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// 16 bytes global -> shared (zeros unless ok), in the background
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// gelu in its tanh form, of the gate, times up
__device__ __forceinline__ float gelu_glu(float gate, float up) {
    return 0.5f * gate * (1.0f + tanhf(0.7978845608028654f * (gate + 0.044715f * gate * gate * gate))) * up;
}

// Tiled TMA load of a 3-D box, completion counted on `bar`
__device__ __forceinline__ void tma_load_3d(uint32_t dst, const CUtensorMap* map, int c0, int c1, int c2, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];"
                 ::"r"(dst), "l"(map), "r"(c0), "r"(c1), "r"(c2), "r"(bar) : "memory");
}

// The ends of a dense linear (scr_dense), applied to one finished f32 sum.
struct DenseEnds {
    void* y;
    float* y2;
    const void* gate;
    long long ldy, y_group, ldy2, ldg;
    int n_main, y_f32, act;
    float limit, alpha;
    float* residual;
    long long ld_residual;
    const float* tanh_w;
    const float* tanh_b;
    float tanh_alpha;
    int n_parts;
    scr_dense_part parts[SCR_DENSE_PARTS];
};
static inline DenseEnds dense_ends(const scr_dense& d) {
    DenseEnds e{d.y, d.y2, d.gate, d.ldy, d.y_group, d.ldy2, d.ldg, d.n_main, d.y_f32, d.act, d.limit, d.alpha,
                d.residual, d.ld_residual, d.tanh_w, d.tanh_b, d.tanh_alpha, d.n_parts, {}};
    for (int p = 0; p < d.n_parts && p < SCR_DENSE_PARTS; ++p) e.parts[p] = d.parts[p];
    return e;
}
// The part column n belongs to and the column the part starts at.
__device__ __forceinline__ int dense_part(const DenseEnds& e, int n, int& start) {
    int p = 0;
    start = 0;
#pragma unroll
    for (int i = 0; i < SCR_DENSE_PARTS - 1; ++i)
        if (i + 1 < e.n_parts && n >= e.parts[i].n_end) {
            p = i + 1;
            start = e.parts[i].n_end;
        }
    return p;
}
// One sum without a residual and parts
template <typename T>
__device__ __forceinline__ void dense_put_own(const DenseEnds& e, int m, int g, int n, float v) {
    if (n >= e.n_main) {
        e.y2[m * e.ldy2 + (n - e.n_main)] = v;
        return;
    }
    const long long col = g * e.y_group + n;
    if (e.gate) v *= sigmoid_f32(to_f32(reinterpret_cast<const T*>(e.gate)[m * e.ldg + col]));
    if (e.y_f32) reinterpret_cast<float*>(e.y)[m * e.ldy + col] = v;
    else reinterpret_cast<T*>(e.y)[m * e.ldy + col] = from_f32<T>(v);
}
template <typename T>
__device__ __forceinline__ void dense_put_residual(const DenseEnds& e, int m, int n, float v) {
    float* r = e.residual + m * e.ld_residual + n;
    v += *r;
    *r = v;
    if (e.tanh_w) reinterpret_cast<T*>(e.y)[m * e.ldy + n] = from_f32<T>(fmaf(tanhf(e.tanh_alpha * v), e.tanh_w[n], e.tanh_b[n]));
}
// The three kinds of ends, an argument of the kernels' templates: a linear's own, several linears in one, the residual.
enum DenseEnd { END_OWN, END_PARTS, END_RESIDUAL };
static inline DenseEnd dense_end(const scr_dense& d) { return d.residual ? END_RESIDUAL : d.n_parts ? END_PARTS : END_OWN; }
template <typename T, DenseEnd END>
__device__ __forceinline__ void dense_put(const DenseEnds& e, int m, int g, int n, float v) {
    if constexpr (END == END_RESIDUAL) {
        dense_put_residual<T>(e, m, n, v);
    } else if constexpr (END == END_PARTS) {
        int start;
        const scr_dense_part& p = e.parts[dense_part(e, n, start)];
        const long long at = m * p.ld + n - start;
        if (p.kind == SCR_PART_F32) reinterpret_cast<float*>(p.y)[at] = v;
        else reinterpret_cast<T*>(p.y)[at] = from_f32<T>(p.kind == SCR_PART_SILU ? v * sigmoid_f32(v) : v);
    } else {
        dense_put_own<T>(e, m, g, n, v);
    }
}
// Columns n (n % 16 < 8) and n + 8 of N.  Where they are a gate and its up they become channel (n / 16) * 8 + n % 8.
template <typename T, DenseEnd END>
__device__ __forceinline__ void dense_put_two(const DenseEnds& e, int m, int g, int n, int N, float a, float b) {
    if (END == END_OWN && e.act) {
        const int c = (n >> 4) * 8 + (n & 7);
        const float v = clamped_glu(a, b, e.limit, e.alpha);
        if (e.y_f32) reinterpret_cast<float*>(e.y)[m * e.ldy + c] = v;
        else reinterpret_cast<T*>(e.y)[m * e.ldy + c] = from_f32<T>(v);
        return;
    }
    if constexpr (END == END_PARTS) {
        int start;
        const scr_dense_part& p = e.parts[dense_part(e, n, start)];
        if (p.kind == SCR_PART_GELU_GLU) {
            const int c = n - start;
            reinterpret_cast<T*>(p.y)[m * p.ld + (c >> 4) * 8 + (c & 7)] = from_f32<T>(gelu_glu(a, b));
            return;
        }
    }
    dense_put<T, END>(e, m, g, n, a);
    if (n + 8 < N) dense_put<T, END>(e, m, g, n + 8, b);
}
