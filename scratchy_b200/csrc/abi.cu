// Workspace query and f32 partial rounding of the quantized-linear C ABI.
#include "common.cuh"
#include <algorithm>

size_t affine_workspace_bytes(int M, int N, int K);
size_t fp8_workspace_bytes(int M, int N, int K);

extern "C" int32_t scr_linear_workspace_size(int32_t kind, int32_t M, int32_t N, int32_t K, size_t* bytes) {
    if (!bytes) return SCR_E_ARG;
    if (M <= 0 || N <= 0 || K <= 0) return SCR_E_SHAPE;
    if (kind == SCR_KIND_AFFINE_B4) { *bytes = affine_workspace_bytes(M, N, K); return SCR_OK; }
    if (kind == SCR_KIND_FP8_DYNAMIC) { *bytes = fp8_workspace_bytes(M, N, K); return SCR_OK; }
    return SCR_E_ARG;
}

__global__ void partial_to_bf16_kernel(const float* __restrict__ in, long long count, uint16_t* __restrict__ out) {
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < count; i += (long long)gridDim.x * blockDim.x) {
        const __nv_bfloat16 v = __float2bfloat16_rn(in[i]);
        out[i] = *reinterpret_cast<const uint16_t*>(&v);
    }
}

extern "C" int32_t scr_partial_to_bf16(scr_ctx* ctx, const float* in, int64_t count, uint16_t* out, void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!in || !out) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (count <= 0) return SCR_OK;
    const int threads = 256;
    const int blocks = (int)std::min<long long>((count + threads - 1) / threads, (long long)ctx->sm_count * 8);
    partial_to_bf16_kernel<<<blocks, threads, 0, (cudaStream_t)stream>>>(in, (long long)count, out);
    return scr_check_launch(ctx, "partial_to_bf16");
}
