// bf16 GEMM on tcgen05 tensor cores for more than 16 rows: y = x W^T, f32 accumulators in TMEM, the ends of `scr_dense`
// in the epilogue.
//
// Persistent, warp-specialised CTA (192 threads), one per SM; a tile is 128 rows of x by BN (128 or 256) rows of W:
//   warp 0     producer: tiled TMA loads of 64-wide k slices of both operands (128-byte swizzle, zero fill outside) into
//              a shared-memory ring; no multicast
//   warp 1     owns TMEM; one thread issues tcgen05.mma (kind::f16, 4 x K=16 per slice) and commits the barriers
//   warps 2-5  epilogue: tcgen05.ld of the 128 x BN accumulator (thread = row), the ends, stores
// Two accumulator buffers let the epilogue of a tile overlap the main loop of the next one.  Groups (one weight block
// per head) are a third tensor-map dimension and part of the tile index.  Few tiles: the k extent is split into work
// units as in `tc_plan_units`, whose f32 partial tiles a second kernel sums in order before it applies the ends.
#include "seq_common.cuh"

#include <algorithm>

namespace {

constexpr int DG_THREADS = 192;
constexpr uint32_t DG_A_BYTES = 128 * 128;                   // 128 rows x 64 bf16

template <int BN>
struct DgSmem {
    static constexpr uint32_t kStageBytes = DG_A_BYTES + BN * 128u;
    static constexpr int kStages = BN == 256 ? 4 : 6;
    static constexpr uint32_t kBarOffset = kStages * kStageBytes;
    static constexpr uint32_t kTotal = kBarOffset + 256u + 1024u;
};

struct DgPlan {
    int bn, mt, ntb, tiles, full, ks_tail;
    int n_tail() const { return tiles - full; }
    size_t slab_floats() const { return ks_tail > 1 ? (size_t)ks_tail * n_tail() * (size_t)(128 * bn) : 0; }
};

DgPlan dg_plan(int M, int N, int K, int groups, int sms) {
    DgPlan best{};
    float best_est = 0.0f;
    for (int bn = 256; bn >= 128; bn -= 128) {
        DgPlan p{};
        p.bn = bn;
        p.mt = scr_ceil_div(M, 128);
        p.ntb = scr_ceil_div(N, bn);
        p.tiles = p.mt * p.ntb * groups;
        const float est = tc_plan_units(p.tiles, scr_ceil_div(K, 64), sms, bn == 256 ? 0.30f : 0.20f, &p.full, &p.ks_tail) * (bn == 256 ? 1.0f : 0.67f);
        if (bn == 256 || est < best_est * 0.97f) {
            best = p;
            best_est = est;
        }
        if (N <= 128 && bn == 256) best_est = 1e30f;           // a single narrow tile: never the wide form
    }
    return best;
}

__device__ __forceinline__ uint4 dg_pack8(const float* v) {
    return make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
}

// The residual end: 32 columns of a row of the stream, and their norm
__device__ __forceinline__ void dg_residual32(const DenseEnds& e, int m, int n0, int N, float (&v)[32]) {
    float* r = e.residual + m * e.ld_residual + n0;
    bf16* h = reinterpret_cast<bf16*>(e.y) + m * e.ldy + n0;
    if (n0 + 32 <= N && (reinterpret_cast<uintptr_t>(r) & 15) == 0 && (!e.tanh_w || (reinterpret_cast<uintptr_t>(h) & 15) == 0)) {
#pragma unroll
        for (int j = 0; j < 32; j += 4) {
            float4 x = *reinterpret_cast<const float4*>(r + j);
            v[j] += x.x;
            v[j + 1] += x.y;
            v[j + 2] += x.z;
            v[j + 3] += x.w;
            *reinterpret_cast<float4*>(r + j) = make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]);
        }
        if (!e.tanh_w) return;
#pragma unroll
        for (int j = 0; j < 32; ++j) v[j] = fmaf(tanhf(e.tanh_alpha * v[j]), __ldg(e.tanh_w + n0 + j), __ldg(e.tanh_b + n0 + j));
#pragma unroll
        for (int j = 0; j < 32; j += 8) *reinterpret_cast<uint4*>(h + j) = dg_pack8(v + j);
    } else {
#pragma unroll
        for (int j = 0; j < 32; ++j)
            if (n0 + j < N) dense_put_residual<bf16>(e, m, n0 + j, v[j]);
    }
}

// Several linears in one matrix: 32 columns, inside one part as a rule
__device__ __forceinline__ void dg_parts32(const DenseEnds& e, int m, int n0, int N, float (&v)[32]) {
    int start;
    const int pi = dense_part(e, n0, start);
    const scr_dense_part p = e.parts[pi];
    const bool glu = p.kind == SCR_PART_GELU_GLU;
    if (min(n0 + 32, N) <= p.n_end && (!glu || ((n0 - start) & 15) == 0)) {
        const int size = p.kind == SCR_PART_F32 ? 4 : 2, cols = min(32, N - n0) >> (glu ? 1 : 0);        // columns that come out
        char* dst = reinterpret_cast<char*>(p.y) + (m * p.ld + (glu ? (n0 - start) >> 1 : n0 - start)) * size;
        const bool vec = (reinterpret_cast<uintptr_t>(dst) & 15) == 0;
        if (p.kind == SCR_PART_F32) {
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
                if (vec && j + 4 <= cols) {
                    reinterpret_cast<float4*>(dst)[j >> 2] = make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]);
                } else {
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (j + i < cols) reinterpret_cast<float*>(dst)[j + i] = v[j + i];
                }
            }
            return;
        }
        if (glu) {
#pragma unroll
            for (int j = 0; j < 16; ++j) v[j] = gelu_glu(v[(j >> 3) * 16 + (j & 7)], v[(j >> 3) * 16 + 8 + (j & 7)]);
        } else if (p.kind == SCR_PART_SILU) {
#pragma unroll
            for (int j = 0; j < 32; ++j) v[j] *= sigmoid_f32(v[j]);
        }
#pragma unroll
        for (int j = 0; j < 32; j += 8) {
            if (vec && j + 8 <= cols) {
                reinterpret_cast<uint4*>(dst)[j >> 3] = dg_pack8(v + j);
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i)
                    if (j + i < cols) reinterpret_cast<bf16*>(dst)[j + i] = __float2bfloat16_rn(v[j + i]);
            }
        }
        return;
    }
#pragma unroll
    for (int j = 0; j < 16; ++j) {
        const int c = (j >> 3) * 16 + (j & 7);
        if (n0 + c < N) dense_put_two<bf16, END_PARTS>(e, m, 0, n0 + c, N, v[c], v[c + 8]);
    }
}

// A linear's own end, with 16-byte stores where the destination allows
__device__ __forceinline__ void dg_own32(const DenseEnds& e, int m, int g, int n0, int N, const float (&v)[32]) {
    if (e.act) {
        // columns 0..7 gate, 8..15 up, 16..23 gate, 24..31 up -> channels c0 .. c0 + 16
        const int c0 = (n0 >> 4) * 8;
        float o[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) o[j] = clamped_glu(v[(j >> 3) * 16 + (j & 7)], v[(j >> 3) * 16 + 8 + (j & 7)], e.limit, e.alpha);
        if (!e.y_f32 && n0 + 32 <= N && (e.ldy & 7) == 0 && (reinterpret_cast<uintptr_t>(e.y) & 15) == 0) {
            uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(e.y) + m * e.ldy + c0);
#pragma unroll
            for (int j = 0; j < 2; ++j)
                dst[j] = make_uint4(pack_bf16x2(o[8 * j], o[8 * j + 1]), pack_bf16x2(o[8 * j + 2], o[8 * j + 3]),
                                    pack_bf16x2(o[8 * j + 4], o[8 * j + 5]), pack_bf16x2(o[8 * j + 6], o[8 * j + 7]));
        } else {
#pragma unroll
            for (int j = 0; j < 16; ++j)
                if (n0 + (j >> 3) * 16 + (j & 7) < N) {
                    if (e.y_f32) reinterpret_cast<float*>(e.y)[m * e.ldy + c0 + j] = o[j];
                    else reinterpret_cast<bf16*>(e.y)[m * e.ldy + c0 + j] = __float2bfloat16_rn(o[j]);
                }
        }
        return;
    }
    const long long at = m * e.ldy + g * e.y_group + n0;
    const bool inside = n0 + 32 <= min(N, e.n_main);
    if (inside && e.y_f32 && !e.gate && (at & 3) == 0 && (reinterpret_cast<uintptr_t>(e.y) & 15) == 0) {
        float4* dst = reinterpret_cast<float4*>(reinterpret_cast<float*>(e.y) + at);
#pragma unroll
        for (int j = 0; j < 8; ++j) dst[j] = make_float4(v[4 * j], v[4 * j + 1], v[4 * j + 2], v[4 * j + 3]);
    } else if (inside && !e.y_f32 && !e.gate && (at & 7) == 0 && (reinterpret_cast<uintptr_t>(e.y) & 15) == 0) {
        uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(e.y) + at);
#pragma unroll
        for (int j = 0; j < 4; ++j)
            dst[j] = make_uint4(pack_bf16x2(v[8 * j], v[8 * j + 1]), pack_bf16x2(v[8 * j + 2], v[8 * j + 3]),
                                pack_bf16x2(v[8 * j + 4], v[8 * j + 5]), pack_bf16x2(v[8 * j + 6], v[8 * j + 7]));
    } else {
#pragma unroll
        for (int j = 0; j < 32; ++j)
            if (n0 + j < N) dense_put_own<bf16>(e, m, g, n0 + j, v[j]);
    }
}

// 32 consecutive columns n0.. of row m: the ends
template <DenseEnd END>
__device__ __forceinline__ void dg_store32(const DenseEnds& e, int m, int g, int n0, int N, float (&v)[32]) {
    if constexpr (END == END_RESIDUAL) return dg_residual32(e, m, n0, N, v);
    else if constexpr (END == END_PARTS) return dg_parts32(e, m, n0, N, v);
    else dg_own32(e, m, g, n0, N, v);
}

template <int BN, DenseEnd END>
__global__ void __launch_bounds__(DG_THREADS, 1)
dense_gemm_kernel(const __grid_constant__ CUtensorMap x_map, const __grid_constant__ CUtensorMap w_map, int M, int N, int KT, int MT,
                  int NTB, int groups, int full, int ks_tail, float* __restrict__ slabs, DenseEnds ends, int* __restrict__ status) {
    using S = DgSmem<BN>;
    extern __shared__ uint8_t smem_raw[];
    const uint32_t smem_base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t* smem_gen = smem_raw + (smem_base - smem_u32(smem_raw));
    const uint32_t bar_base = smem_base + S::kBarOffset;
    auto full_bar = [&](int s) { return bar_base + 8u * s; };
    auto empty_bar = [&](int s) { return bar_base + 8u * (S::kStages + s); };
    auto accf_bar = [&](int b) { return bar_base + 8u * (2 * S::kStages + b); };
    auto acce_bar = [&](int b) { return bar_base + 8u * (2 * S::kStages + 2 + b); };
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem_gen + S::kBarOffset + 8 * (2 * S::kStages + 4));

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n_tail = MT * NTB * groups - full;
    const int units = full + n_tail * ks_tail;

    pdl_trigger();
    if (threadIdx.x == 0) {
        for (int s = 0; s < S::kStages; ++s) { mbar_init(full_bar(s), 1); mbar_init(empty_bar(s), 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(accf_bar(b), 1); mbar_init(acce_bar(b), 128); }
        fence_mbar_init();
    }
    if (warp == 1) {
        tmem_alloc(smem_u32((const void*)tmem_slot), 2 * BN);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    pdl_wait();

    if (warp == 0) {
        if (lane == 0) {
            int s = 0;
            uint32_t ph = 0;
            for (int unit = blockIdx.x; unit < units; unit += gridDim.x) {
                int tile, ks, k_lo, k_hi;
                tc_unit(unit, full, ks_tail, KT, tile, ks, k_lo, k_hi);
                const int mt = tile % MT, nb = (tile / MT) % NTB, g = tile / (MT * NTB);
                for (int kt = k_lo; kt < k_hi; ++kt) {
                    mbar_wait(empty_bar(s), ph ^ 1u, status, TC_ERR_EMPTY_WAIT);
                    const uint32_t sa = smem_base + s * S::kStageBytes;
                    mbar_arrive_expect_tx(full_bar(s), S::kStageBytes);
                    tma_load_3d(sa, &x_map, kt * 64, g, mt * 128, full_bar(s));
                    tma_load_3d(sa + DG_A_BYTES, &w_map, kt * 64, nb * BN, g, full_bar(s));
                    if (++s == S::kStages) { s = 0; ph ^= 1u; }
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = umma_idesc(1, 1, 128, BN);
            int s = 0, it = 0;
            uint32_t ph = 0;
            for (int unit = blockIdx.x; unit < units; unit += gridDim.x, ++it) {
                int tile, ks, k_lo, k_hi;
                tc_unit(unit, full, ks_tail, KT, tile, ks, k_lo, k_hi);
                const int buf = it & 1;
                mbar_wait(acce_bar(buf), ((uint32_t)(it >> 1) & 1u) ^ 1u, status, TC_ERR_ACC_EMPTY);
                tc_fence_after();
                const uint32_t d_tmem = tmem_base + (uint32_t)(buf * BN);
                for (int kt = k_lo; kt < k_hi; ++kt) {
                    mbar_wait(full_bar(s), ph, status, TC_ERR_FULL_WAIT);
                    tc_fence_after();
                    const uint32_t sa = smem_base + s * S::kStageBytes;
                    const uint64_t adesc = umma_desc_k_sw128(sa), bdesc = umma_desc_k_sw128(sa + DG_A_BYTES);
#pragma unroll
                    for (int k4 = 0; k4 < 4; ++k4)
                        umma_f16(d_tmem, adesc + (uint64_t)(2 * k4), bdesc + (uint64_t)(2 * k4), idesc, ((kt - k_lo) | k4) != 0);
                    umma_commit(empty_bar(s));
                    if (++s == S::kStages) { s = 0; ph ^= 1u; }
                }
                umma_commit(accf_bar(buf));
            }
        }
    } else {
        const int q = warp & 3;
        int it = 0;
        for (int unit = blockIdx.x; unit < units; unit += gridDim.x, ++it) {
            int tile, ks, k_lo, k_hi;
            tc_unit(unit, full, ks_tail, KT, tile, ks, k_lo, k_hi);
            const int mt = tile % MT, nb = (tile / MT) % NTB, g = tile / (MT * NTB);
            const int buf = it & 1, m = mt * 128 + q * 32 + lane;
            const bool split = unit >= full && ks_tail > 1;
            float* slab = split ? slabs + ((size_t)ks * n_tail + (tile - full)) * (size_t)(128 * BN) + (size_t)(q * 32 + lane) * BN : nullptr;
            mbar_wait(accf_bar(buf), (uint32_t)(it >> 1) & 1u, status, TC_ERR_ACC_FULL);
            tc_fence_after();
            for (int c = 0; c < BN / 32; ++c) {
                const int n0 = nb * BN + c * 32;
                if (n0 >= N) break;
                uint32_t r[32];
                tmem_ld_32x32(tmem_base + ((uint32_t)(q * 32) << 16) + (uint32_t)(buf * BN + c * 32), r);
                tmem_ld_wait();
                if (m >= M) continue;
                if (split) {
                    float4* dst = reinterpret_cast<float4*>(slab + c * 32);
#pragma unroll
                    for (int j = 0; j < 8; ++j)
                        dst[j] = make_float4(__uint_as_float(r[4 * j]), __uint_as_float(r[4 * j + 1]), __uint_as_float(r[4 * j + 2]), __uint_as_float(r[4 * j + 3]));
                } else {
                    float v[32];
#pragma unroll
                    for (int j = 0; j < 32; ++j) v[j] = __uint_as_float(r[j]);
                    dg_store32<END>(ends, m, g, n0, N, v);
                }
            }
            tc_fence_before();
            mbar_arrive(acce_bar(buf));
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, 2 * BN);
    }
}

// Sums a split tile's partial tiles in order and applies the ends: one thread per row and 32 columns would leave most
// of the GPU idle on few rows, so one thread takes a gate column and its up column (16-column runs: j and j + 8).
template <DenseEnd END>
__global__ void __launch_bounds__(256) dense_gemm_finish_kernel(const float* __restrict__ slabs, int ks_tail, int n_tail, int full, int MT,
                                                                int NTB, int bn, int M, int N, DenseEnds ends) {
    pdl_trigger();
    pdl_wait();
    const int per_row = bn / 2, rows_per_cta = 256 / per_row, blocks_per_tile = 128 / rows_per_cta;
    const int tt = blockIdx.x / blocks_per_tile, tile = full + tt;
    const int mt = tile % MT, nb = (tile / MT) % NTB, g = tile / (MT * NTB);
    const int rl = (blockIdx.x % blocks_per_tile) * rows_per_cta + threadIdx.x / per_row, p = threadIdx.x % per_row;
    const int c = (p >> 3) * 16 + (p & 7), m = mt * 128 + rl, n = nb * bn + c;
    if (m >= M || n >= N) return;
    const size_t tile_elems = (size_t)128 * bn;
    const float* src = slabs + (size_t)tt * tile_elems + (size_t)rl * bn + c;
    float a = 0.0f, b = 0.0f;
    for (int k = 0; k < ks_tail; ++k) {
        a += src[(size_t)k * n_tail * tile_elems];
        b += src[(size_t)k * n_tail * tile_elems + 8];
    }
    dense_put_two<bf16, END>(ends, m, g, n, N, a, b);
}

bool dg_map(CUtensorMap* map, const void* base, uint64_t d0, uint64_t d1, uint64_t d2, uint64_t s1, uint64_t s2, uint32_t b1, uint32_t b2) {
    tc_encode_tiled_fn enc = tc_tensor_map_encoder();
    if (!enc) return false;
    const cuuint64_t dims[3] = {d0, d1, d2};
    const cuuint64_t strides[2] = {s1, s2};
    const cuuint32_t box[3] = {64, b1, b2}, one[3] = {1, 1, 1};
    return enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE,
               CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int BN, DenseEnd END>
int32_t dg_launch(scr_ctx* ctx, const scr_dense& d, const DgPlan& p, float* slabs, cudaStream_t stream) {
    CUtensorMap x_map, w_map;
    const uint64_t xg = d.groups > 1 ? (uint64_t)d.x_group * 2 : (uint64_t)d.K * 2;
    if (!dg_map(&x_map, d.x, d.K, d.groups, d.M, xg, (uint64_t)d.ldx * 2, 1, 128) ||
        !dg_map(&w_map, d.w, d.K, d.N, d.groups, (uint64_t)d.K * 2, (uint64_t)d.N * d.K * 2, BN, 1))
        return scr_fail(ctx, SCR_E_CUDA, "dense_gemm: tensor map (M %d N %d K %d groups %d)", d.M, d.N, d.K, d.groups);
    cudaError_t e = seq_smem(dense_gemm_kernel<BN, END>, DgSmem<BN>::kTotal);
    if (e == cudaSuccess) {
        const int units = p.full + p.n_tail() * p.ks_tail;
        e = launch_pdl(dense_gemm_kernel<BN, END>, dim3(std::min(units, ctx->sm_count)), dim3(DG_THREADS), DgSmem<BN>::kTotal, stream, x_map, w_map, d.M,
                       d.N, scr_ceil_div(d.K, 64), p.mt, p.ntb, d.groups, p.full, p.ks_tail, slabs, dense_ends(d), ctx->dev_status);
    }
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "dense_gemm: %s", cudaGetErrorString(e));
    const int32_t st = scr_check_launch(ctx, "dense_gemm");
    if (st || p.ks_tail == 1) return st;
    e = launch_pdl(dense_gemm_finish_kernel<END>, dim3(p.n_tail() * (128 / (512 / BN))), dim3(256), 0, stream, (const float*)slabs, p.ks_tail, p.n_tail(),
                   p.full, p.mt, p.ntb, BN, d.M, d.N, dense_ends(d));
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "dense_gemm_finish: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "dense_gemm_finish");
}

}  // namespace

size_t dense_gemm_workspace(int M, int N, int K, int groups) { return dg_plan(M, N, K, groups, tc_sm_count()).slab_floats() * sizeof(float); }

int32_t dense_gemm_launch(scr_ctx* ctx, const scr_dense& d, void* workspace, size_t workspace_bytes, cudaStream_t stream) {
    const DgPlan p = dg_plan(d.M, d.N, d.K, d.groups, ctx->sm_count);
    if (p.slab_floats() * sizeof(float) > workspace_bytes || (p.ks_tail > 1 && (!workspace || !scr_aligned16(workspace))))
        return scr_fail(ctx, SCR_E_WORKSPACE, "dense_gemm needs %zu bytes of workspace", p.slab_floats() * sizeof(float));
    float* slabs = (float*)workspace;
#define DG_CASE(END) case END: return p.bn == 256 ? dg_launch<256, END>(ctx, d, p, slabs, stream) : dg_launch<128, END>(ctx, d, p, slabs, stream)
    switch (dense_end(d)) {
        DG_CASE(END_PARTS);
        DG_CASE(END_RESIDUAL);
        default: DG_CASE(END_OWN);
    }
#undef DG_CASE
}
