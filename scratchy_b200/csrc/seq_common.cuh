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

// The ends of a dense linear (scr_dense), applied to one finished f32 sum.
struct DenseEnds {
    void* y;
    float* y2;
    const void* gate;
    long long ldy, y_group, ldy2, ldg;
    int n_main, y_f32, act;
    float limit, alpha;
};
static inline DenseEnds dense_ends(const scr_dense& d) {
    return DenseEnds{d.y, d.y2, d.gate, d.ldy, d.y_group, d.ldy2, d.ldg, d.n_main, d.y_f32, d.act, d.limit, d.alpha};
}
template <typename T>
__device__ __forceinline__ void dense_put(const DenseEnds& e, int m, int g, int n, float v) {
    if (n >= e.n_main) {
        e.y2[m * e.ldy2 + (n - e.n_main)] = v;
        return;
    }
    const long long col = g * e.y_group + n;
    if (e.gate) v *= sigmoid_f32(to_f32(reinterpret_cast<const T*>(e.gate)[m * e.ldg + col]));
    if (e.y_f32) reinterpret_cast<float*>(e.y)[m * e.ldy + col] = v;
    else reinterpret_cast<T*>(e.y)[m * e.ldy + col] = from_f32<T>(v);
}
// act 1: the gate row n (n % 16 < 8) and its up row n + 8 become channel (n / 16) * 8 + n % 8
template <typename T>
__device__ __forceinline__ void dense_put_pair(const DenseEnds& e, int m, int n, float gate, float up) {
    const int c = (n >> 4) * 8 + (n & 7);
    const float v = clamped_glu(gate, up, e.limit, e.alpha);
    if (e.y_f32) reinterpret_cast<float*>(e.y)[m * e.ldy + c] = v;
    else reinterpret_cast<T*>(e.y)[m * e.ldy + c] = from_f32<T>(v);
}
