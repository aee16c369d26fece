// Full-precision linears of the sequence models: y = x W^T with the ends of `scr_dense`.
//
//   M <= 16, bf16   dense_matvec_kernel   weights streamed once from HBM straight into mma.sync fragments (decode)
//   M > 16, bf16    dense_gemm.cu         tcgen05 GEMM
//   otherwise       dense_plain_kernel    f32 arithmetic on any sizes (the f32 data type; bf16 rows that are not a
//                                         multiple of 16 bytes)
#include "seq_common.cuh"

#include <algorithm>

size_t dense_gemm_workspace(int M, int N, int K, int groups);
int32_t dense_gemm_launch(scr_ctx* ctx, const scr_dense& d, void* workspace, size_t workspace_bytes, cudaStream_t stream);

namespace {

// ------------------------------------------------------------------------------- any size, f32 arithmetic
// 64 rows x 64 columns per CTA, 4 x 4 per thread.  A thread's columns are 8 apart, so a gate column and its up column
// (8 further on) belong to one thread.
constexpr int PLAIN_T = 64, PLAIN_K = 16;

template <typename T, DenseEnd END>
__global__ void __launch_bounds__(256) dense_plain_kernel(const T* __restrict__ w, const T* __restrict__ x, long long ldx,
                                                          long long x_group, int M, int N, int K, DenseEnds ends) {
    __shared__ float xs[PLAIN_K][PLAIN_T + 4], ws[PLAIN_K][PLAIN_T + 4];
    pdl_trigger();
    pdl_wait();
    const int g = blockIdx.z, m0 = blockIdx.y * PLAIN_T, n0 = blockIdx.x * PLAIN_T;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const int cbase = (tx >> 3) * 32 + (tx & 7);
    w += (size_t)g * N * K;
    x += g * x_group;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += PLAIN_K) {
        for (int i = threadIdx.x; i < PLAIN_T * PLAIN_K; i += 256) {
            const int r = i >> 4, k = i & 15;
            xs[k][r] = (m0 + r < M && k0 + k < K) ? to_f32(x[(m0 + r) * ldx + k0 + k]) : 0.0f;
            ws[k][r] = (n0 + r < N && k0 + k < K) ? to_f32(w[(size_t)(n0 + r) * K + k0 + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < PLAIN_K; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[i] = xs[k][ty * 4 + i];
                b[i] = ws[k][cbase + 8 * i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; j += 2)
            if (n0 + cbase + 8 * j < N) dense_put_two<T, END>(ends, m, g, n0 + cbase + 8 * j, N, acc[i][j], acc[i][j + 1]);
    }
}

// ------------------------------------------------------------------------------- decode matvec
// A tile is 16 weight rows over the whole K, shared by `wpt` warps of each CTA of a cluster, which take 64-wide units of K
// in turn.  In a unit lane (g, t) loads the 16-byte pieces [t*8, t*8+8) and [32 + t*8, ..) of rows g and g + 8, and the
// same pieces of activation row g: the k order inside a fragment is a permutation both operands share, so the loaded
// registers are mma operands as they stand (weights = A, 8 tokens per B).  A warp keeps SLOTS units in flight and refills a
// unit's registers as soon as they are used; the first ones, load-time constants, are requested before the wait for the
// preceding kernel.  Partial sums meet in shared memory in warp order, then in the cluster's first CTA in rank order.
constexpr int MV_WARPS = 8, MV_MAX_CLUSTER = 4;

__device__ __forceinline__ uint32_t mv_cluster_rank() {
    uint32_t r;
    asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}

template <int NT, int SLOTS, DenseEnd END>
__global__ void __launch_bounds__(MV_WARPS * 32, 2) dense_matvec_kernel(const bf16* __restrict__ w, const bf16* __restrict__ x,
                                                                        long long ldx, long long x_group, int M, int N, int K,
                                                                        int wpt, int cluster, DenseEnds ends) {
    __shared__ float red[MV_WARPS][16][8 * NT + 1];
    __shared__ float peers[MV_MAX_CLUSTER - 1][MV_WARPS][16][8 * NT];          // [rank - 1][tile][row][token], filled on rank 0
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int rank = cluster > 1 ? (int)mv_cluster_rank() : 0;
    const int tiles = MV_WARPS / wpt, part = warp % wpt + rank * wpt, step = wpt * cluster, grp = blockIdx.y;
    const int tile0 = (blockIdx.x / cluster) * tiles;
    const int n0 = (tile0 + warp / wpt) * 16;
    const int units = (K + 63) >> 6;
    const bf16* w0 = w + ((size_t)grp * N + min(n0 + g, N - 1)) * K + t * 8;
    const bf16* w1 = w + ((size_t)grp * N + min(n0 + g + 8, N - 1)) * K + t * 8;
    x += grp * x_group + t * 8;
    uint4 wa[SLOTS][2], wb[SLOTS][2], xv[SLOTS][2][NT];
    const uint4 zero = make_uint4(0, 0, 0, 0);
    auto load_w = [&](int s, int u) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int k = u * 64 + h * 32;
            const bool ok = k + t * 8 < K;
            wa[s][h] = ok ? ld_stream_v4(w0 + k) : zero;
            wb[s][h] = ok ? ld_stream_v4(w1 + k) : zero;
        }
    };
    auto load_x = [&](int s, int u) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int k = u * 64 + h * 32;
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) xv[s][h][nt] = (nt * 8 + g < M && k + t * 8 < K) ? ld_act_v4(x + (nt * 8 + g) * ldx + k) : zero;
        }
    };
    float acc[NT][4] = {};
#pragma unroll
    for (int s = 0; s < SLOTS; ++s) load_w(s, part + s * step);
    pdl_wait();
#pragma unroll
    for (int s = 0; s < SLOTS; ++s) load_x(s, part + s * step);
    for (int u0 = part; u0 < units; u0 += SLOTS * step) {
#pragma unroll
        for (int s = 0; s < SLOTS; ++s) {
#pragma unroll
            for (int h = 0; h < 2; ++h)
#pragma unroll
                for (int nt = 0; nt < NT; ++nt) {
                    mma_16816(acc[nt], wa[s][h].x, wb[s][h].x, wa[s][h].y, wb[s][h].y, xv[s][h][nt].x, xv[s][h][nt].y);
                    mma_16816(acc[nt], wa[s][h].z, wb[s][h].z, wa[s][h].w, wb[s][h].w, xv[s][h][nt].z, xv[s][h][nt].w);
                }
            load_w(s, u0 + (s + SLOTS) * step);
            load_x(s, u0 + (s + SLOTS) * step);
        }
    }
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
        red[warp][g][nt * 8 + 2 * t] = acc[nt][0];
        red[warp][g][nt * 8 + 2 * t + 1] = acc[nt][1];
        red[warp][g + 8][nt * 8 + 2 * t] = acc[nt][2];
        red[warp][g + 8][nt * 8 + 2 * t + 1] = acc[nt][3];
    }
    __syncthreads();
    auto total = [&](int tile, int r, int m) {
        float v = 0.0f;
        for (int p = 0; p < wpt; ++p) v += red[tile * wpt + p][r][m];
        return v;
    };
    if (cluster > 1) {
        if (rank > 0) {
            for (int i = threadIdx.x; i < tiles * 16 * M; i += MV_WARPS * 32) {
                const int r = i & 15, tile = (i >> 4) % tiles, m = (i >> 4) / tiles;
                uint32_t dst;
                asm volatile("mapa.shared::cluster.u32 %0, %1, 0;" : "=r"(dst) : "r"(smem_u32(&peers[rank - 1][tile][r][m])));
                asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(total(tile, r, m)) : "memory");
            }
        }
        asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
        if (rank > 0) return;
    }
    auto whole = [&](int tile, int r, int m) {
        float v = total(tile, r, m);
        for (int c = 1; c < cluster; ++c) v += peers[c - 1][tile][r][m];
        return v;
    };
    if (END == END_PARTS || (END == END_OWN && ends.act)) {
        for (int i = threadIdx.x; i < tiles * 8 * M; i += MV_WARPS * 32) {
            const int r = i & 7, tile = (i >> 3) % tiles, m = (i >> 3) / tiles;
            const int n = (tile0 + tile) * 16 + r;
            if (n < N) dense_put_two<bf16, END>(ends, m, grp, n, N, whole(tile, r, m), whole(tile, r + 8, m));
        }
    } else {
        for (int i = threadIdx.x; i < tiles * 16 * M; i += MV_WARPS * 32) {
            const int r = i & 15, tile = (i >> 4) % tiles, m = (i >> 4) / tiles;
            const int n = (tile0 + tile) * 16 + r;
            if (n < N) dense_put<bf16, END>(ends, m, grp, n, whole(tile, r, m));
        }
    }
}

template <DenseEnd END>
int32_t matvec_launch(scr_ctx* ctx, const scr_dense& d, cudaStream_t stream) {
    const int units = (d.K + 63) / 64, tiles16 = (d.N + 15) / 16;
    // warps per tile: enough units of K for each, and enough CTAs to fill the GPU
    int wpt = 1;
    while (wpt < MV_WARPS && (units >= 4 * wpt || (units >= 2 * wpt && (tiles16 * d.groups * wpt) / MV_WARPS < 2 * ctx->sm_count))) wpt *= 2;
    const int blocks = scr_ceil_div(tiles16, MV_WARPS / wpt);
    // fewer, long tiles than SMs: a cluster shares each
    int cluster = 1;
    while (cluster < MV_MAX_CLUSTER && blocks * d.groups * cluster < ctx->sm_count && units >= 16 * wpt * cluster) cluster *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(blocks * cluster, d.groups);
    cfg.blockDim = dim3(MV_WARPS * 32);
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = cluster > 1 ? 2 : 1;
    const bf16 *w = (const bf16*)d.w, *x = (const bf16*)d.x;
    const long long ldx = d.ldx, xg = d.x_group;
    const DenseEnds e = dense_ends(d);
    const cudaError_t err = d.M <= 8 ? cudaLaunchKernelEx(&cfg, dense_matvec_kernel<1, 3, END>, w, x, ldx, xg, d.M, d.N, d.K, wpt, cluster, e)
                                     : cudaLaunchKernelEx(&cfg, dense_matvec_kernel<2, 2, END>, w, x, ldx, xg, d.M, d.N, d.K, wpt, cluster, e);
    if (err != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "dense_matvec: %s", cudaGetErrorString(err));
    return scr_check_launch(ctx, "dense_matvec");
}

template <typename T>
int32_t plain_launch(scr_ctx* ctx, const scr_dense& d, cudaStream_t stream) {
    const dim3 grid(scr_ceil_div(d.N, PLAIN_T), scr_ceil_div(d.M, PLAIN_T), d.groups);
    const DenseEnd end = dense_end(d);
    auto kernel = end == END_RESIDUAL ? dense_plain_kernel<T, END_RESIDUAL> : end == END_PARTS ? dense_plain_kernel<T, END_PARTS> : dense_plain_kernel<T, END_OWN>;
    const cudaError_t err = launch_pdl(kernel, grid, dim3(256), 0, stream, (const T*)d.w, (const T*)d.x,
                                       (long long)d.ldx, (long long)d.x_group, d.M, d.N, d.K, dense_ends(d));
    if (err != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "dense_plain: %s", cudaGetErrorString(err));
    return scr_check_launch(ctx, "dense_plain");
}

bool rows_of_16_bytes(const scr_dense& d) {
    return d.K % 8 == 0 && d.ldx % 8 == 0 && d.x_group % 8 == 0 && scr_aligned16(d.w) && scr_aligned16(d.x);
}

}  // namespace

extern "C" int32_t scr_dense_workspace_size(int32_t dtype, int32_t M, int32_t N, int32_t K, int32_t groups, size_t* bytes) {
    if (!bytes) return SCR_E_ARG;
    if (M <= 0 || N <= 0 || K <= 0 || groups <= 0) return SCR_E_SHAPE;
    *bytes = (dtype == SCR_DTYPE_BF16 && M > 16) ? dense_gemm_workspace(M, N, K, groups) : 0;
    return SCR_OK;
}

extern "C" int32_t scr_dense_linear(scr_ctx* ctx, int32_t dtype, const scr_dense* dp, void* workspace, size_t workspace_bytes,
                                    void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!dp || !dp->w || !dp->x) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    const scr_dense& d = *dp;
    if (!d.y && !d.n_parts && (!d.residual || d.tanh_w)) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (d.residual && (d.groups != 1 || d.n_parts || d.act || d.gate || d.n_main < d.N || (d.tanh_w && !d.tanh_b)))
        return scr_fail(ctx, SCR_E_ARG, "a residual end stands alone");
    if (d.n_parts < 0 || d.n_parts > SCR_DENSE_PARTS) return scr_fail(ctx, SCR_E_ARG, "%d parts", d.n_parts);
    for (int p = 0, start = 0; p < d.n_parts; start = d.parts[p++].n_end) {
        const scr_dense_part& q = d.parts[p];
        if (!q.y || q.kind < SCR_PART_STORE || q.kind > SCR_PART_GELU_GLU) return scr_fail(ctx, SCR_E_ARG, "part %d", p);
        if (q.n_end <= start || (p + 1 == d.n_parts && q.n_end != d.N) || d.groups != 1 || d.act || d.gate)
            return scr_fail(ctx, SCR_E_SHAPE, "parts cover the columns of one group in order");
        if (q.kind == SCR_PART_GELU_GLU && (start % 16 || q.n_end % 16)) return scr_fail(ctx, SCR_E_SHAPE, "gate/up pairs come in runs of 8 + 8 rows");
    }
    if (d.M <= 0 || d.N <= 0 || d.K <= 0 || d.groups <= 0) return scr_fail(ctx, SCR_E_SHAPE, "empty linear (M %d N %d K %d)", d.M, d.N, d.K);
    if (!d.n_parts && d.n_main < d.N && (!d.y2 || d.groups != 1 || d.act)) return scr_fail(ctx, SCR_E_ARG, "a second output needs y2, one group and no activation");
    if (d.act && (d.N % 16 || d.groups != 1 || d.gate)) return scr_fail(ctx, SCR_E_SHAPE, "gate/up pairs come in runs of 8 + 8 rows");
    cudaStream_t st = (cudaStream_t)stream;
    if (dtype == SCR_DTYPE_F32) return plain_launch<float>(ctx, d, st);
    if (dtype != SCR_DTYPE_BF16) return scr_fail(ctx, SCR_E_DTYPE, "dtype %d", dtype);
    if (!rows_of_16_bytes(d)) return plain_launch<bf16>(ctx, d, st);
    if (d.M <= 16)
        return d.residual ? matvec_launch<END_RESIDUAL>(ctx, d, st) : d.n_parts ? matvec_launch<END_PARTS>(ctx, d, st) : matvec_launch<END_OWN>(ctx, d, st);
    return dense_gemm_launch(ctx, d, workspace, workspace_bytes, st);
}
