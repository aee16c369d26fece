// Latent attention for decoding and short portions, bf16, on mma.sync: the rows of a sequence are its tokens x heads, all
// of which read the same cache rows [latent | rotated key part].
//
// A CTA takes 16 or 32 of those rows and a share of the keys.  Key tiles of 64 cache rows come through two shared-memory
// stages (cp.async, one warp per row of the paged cache, the next tile in flight while this one is computed, its rows'
// addresses looked up a tile earlier).  Per tile: S = Q K^T with warp = (quarter of the dimensions, half of the keys), so
// that a warp keeps its part of Q in registers and every key element is read once; the quarters meet in shared memory in
// f32; a softmax pass over the rows that keeps the running maximum and sum in f32 and leaves P as a bf16 head and
// remainder (two products, so the weights keep about 16 bits); O += P V with the latent columns dealt to the warps, V
// being the first kv_rank columns of the very tile.
// Shares of the keys that other CTAs took meet in a second kernel.
#include "seq_common.cuh"

#include <algorithm>

namespace {

constexpr int LM_THREADS = 256, LM_KEYS = 64, LM_P_LD = LM_KEYS + 8, LM_S_LD = LM_KEYS + 4;

struct LmSmem {
    int ld;                                                    // elements per row of Q and key tiles: odd multiple of 16 bytes
    size_t q, tile, scores, p_hi, p_lo, corr, total;
    static __host__ __device__ LmSmem of(int D, int mt) {
        LmSmem s{};
        s.ld = (D + 15) / 16 * 16 + 8;
        s.q = s.scores = 0;                                    // Q moves to registers before the first scores are written
        const size_t q = (size_t)mt * 16 * s.ld * 2, part = 4 * (size_t)mt * 16 * LM_S_LD * 4;
        s.tile = q > part ? q : part;
        s.p_hi = s.tile + 2 * (size_t)LM_KEYS * s.ld * 2;
        s.p_lo = s.p_hi + (size_t)mt * 16 * LM_P_LD * 2;
        s.corr = s.p_lo + (size_t)mt * 16 * LM_P_LD * 2;
        s.total = s.corr + (size_t)mt * 16 * 4 * 2;
        return s;
    }
};

// MT: 16-row tiles; NTW: 8-column tiles of the latent per warp (kv_rank <= 64 * NTW, kv_rank + rot_dim <= 64 * (NTW + 1))
template <int MT, int NTW>
__global__ void __launch_bounds__(LM_THREADS) latent_attention_mma_kernel(scr_latent_shape s, scr_step st, const bf16* __restrict__ q,
                                                                          const bf16* __restrict__ cache, bf16* __restrict__ out,
                                                                          float* __restrict__ part_o, float* __restrict__ part_ml, int nsplit,
                                                                          int* __restrict__ status) {
    extern __shared__ __align__(128) unsigned char lm_smem[];
    constexpr int ROWS = MT * 16, TPR = LM_THREADS / ROWS, KPT = LM_KEYS / TPR;      // softmax: threads per row, keys per thread
    const int D = s.kv_rank + s.rot_dim;
    const LmSmem lay = LmSmem::of(D, MT);
    bf16* Q = reinterpret_cast<bf16*>(lm_smem + lay.q);
    float* scores = reinterpret_cast<float*>(lm_smem + lay.scores);
    bf16* p_hi = reinterpret_cast<bf16*>(lm_smem + lay.p_hi);
    bf16* p_lo = reinterpret_cast<bf16*>(lm_smem + lay.p_lo);
    float* corr = reinterpret_cast<float*>(lm_smem + lay.corr);                      // [ROWS] rescale, then [ROWS] final sums
    pdl_trigger();
    const int b = blockIdx.z, split = blockIdx.y, r0 = blockIdx.x * ROWS;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int first = st.segs[b * 4], count = st.segs[b * 4 + 1], pos0 = st.segs[b * 4 + 2];
    const int nrows = min(ROWS, count * s.heads - r0);
    if (nrows <= 0 || first < 0 || first + count > st.rows) { pdl_wait(); return; }
    int kv = pos0 + (r0 + nrows - 1) / s.heads + 1;                                  // keys the last row of this CTA sees
    if (kv > s.max_blocks * s.block_size) {
        if (threadIdx.x == 0) atomicCAS(status, 0, SEQ_BAD_POSITION);
        kv = s.max_blocks * s.block_size;
    }
    const int tiles = (kv + LM_KEYS - 1) / LM_KEYS, per = (tiles + nsplit - 1) / nsplit;
    const int t_lo = min(split * per, tiles), t_hi = min(t_lo + per, tiles);
    const int* table = st.block_table + (size_t)b * s.max_blocks;
    const int chunks = D / 8;
    constexpr int RPW = LM_KEYS / 8;                                                 // key rows a warp loads per tile
    // lane i of a warp: where row i of the warp's share of tile t lives in the cache, -1 outside
    auto look_up = [&](int t) {
        const int key = t * LM_KEYS + warp * RPW + (lane & (RPW - 1));
        if (t >= t_hi || key >= kv) return -1ll;
        const int blk = key / s.block_size, block = table[blk];
        if (block < 0 || block >= s.num_blocks) {
            atomicCAS(status, 0, SEQ_BAD_BLOCK);
            return -1ll;
        }
        return ((long long)block * s.block_size + (key - blk * s.block_size)) * D;
    };
    auto load_tile = [&](int t, long long where) {
        bf16* dst = reinterpret_cast<bf16*>(lm_smem + lay.tile) + (size_t)((t - t_lo) & 1) * LM_KEYS * lay.ld;
#pragma unroll
        for (int i = 0; i < RPW; ++i) {
            const long long off = __shfl_sync(0xffffffffu, where, i);
            const bf16* src = cache + (off < 0 ? 0 : off);
            const uint32_t row = smem_u32(dst + (size_t)(warp * RPW + i) * lay.ld);
            for (int c = lane; c < chunks; c += 32) cp_async16(row + c * 16, src + c * 8, off >= 0);
        }
    };
    // zero what a key row holds beyond D (the last k step may read it), in both stages and in Q
    for (int i = threadIdx.x; i < (2 * LM_KEYS + ROWS) * (lay.ld - D); i += LM_THREADS) {
        const int row = i / (lay.ld - D), c = D + i % (lay.ld - D);
        (row < ROWS ? Q + (size_t)row * lay.ld : reinterpret_cast<bf16*>(lm_smem + lay.tile) + (size_t)(row - ROWS) * lay.ld)[c] = __float2bfloat16_rn(0.0f);
    }
    // cache rows before this step's are there already: their tile does not wait for the preceding kernels
    const bool early = t_lo < t_hi && (t_lo + 1) * LM_KEYS <= pos0;
    if (early) load_tile(t_lo, look_up(t_lo));
    pdl_wait();
    if (!early && t_lo < t_hi) load_tile(t_lo, look_up(t_lo));
    long long where_next = look_up(t_lo + 1);
    for (int i = threadIdx.x; i < ROWS * chunks; i += LM_THREADS) {
        const int row = i / chunks, c = i - row * chunks;
        cp_async16(smem_u32(Q + (size_t)row * lay.ld + c * 8), q + ((size_t)first * s.heads + r0 + (row < nrows ? row : 0)) * D + c * 8, row < nrows);
    }
    cp_async_commit();

    float acc[MT][NTW][4] = {};
    const float sl2 = s.scale * 1.4426950408889634f;
    const int srow = threadIdx.x / TPR, sk0 = (threadIdx.x % TPR) * 4;               // this thread's softmax row; its keys: runs of 4, 4 * TPR apart
    const int limit = pos0 + (r0 + min(srow, nrows - 1)) / s.heads;                  // last key the row sees
    float m_run = -INFINITY, l_run = 0.0f;
    constexpr int KQ = NTW + 1;                                                      // k steps of 16 per quarter of the dimensions
    const int kq = warp & 3, kh = warp >> 2;                                         // S phase: quarter of the dimensions, half of the keys
    const int k_lo = kq * KQ, k_n = min(KQ, (D + 15) / 16 - k_lo), lm = lane >> 3, lr = lane & 7;   // (zero from D up to ld)
    uint32_t qf[MT][KQ][4];
    cp_async_wait_all();
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int k = 0; k < KQ; ++k) {
            qf[m][k][0] = qf[m][k][1] = qf[m][k][2] = qf[m][k][3] = 0;
            if (k < k_n) ldsm_x4(smem_u32(Q + (size_t)(m * 16 + (lm & 1) * 8 + lr) * lay.ld + (k_lo + k) * 16 + (lm >> 1) * 8), qf[m][k]);
        }
    for (int t = t_lo; t < t_hi; ++t) {
        cp_async_wait_all();
        __syncthreads();
        if (t + 1 < t_hi) load_tile(t + 1, where_next);
        cp_async_commit();
        where_next = look_up(t + 2);
        const bf16* K = reinterpret_cast<bf16*>(lm_smem + lay.tile) + (size_t)((t - t_lo) & 1) * LM_KEYS * lay.ld;
        {
            float sc[MT][4][4] = {};
            const uint32_t kb = smem_u32(K + (size_t)(kh * 32 + (lm >> 1) * 8 + lr) * lay.ld + k_lo * 16 + (lm & 1) * 8);
#pragma unroll
            for (int k = 0; k < KQ; ++k) {
                if (k < k_n) {
                    uint32_t kf[2][4];
#pragma unroll
                    for (int n2 = 0; n2 < 2; ++n2) ldsm_x4(kb + (uint32_t)(n2 * 16 * lay.ld * 2) + k * 32, kf[n2]);
#pragma unroll
                    for (int m = 0; m < MT; ++m)
#pragma unroll
                        for (int n = 0; n < 4; ++n)
                            mma_16816(sc[m][n], qf[m][k][0], qf[m][k][1], qf[m][k][2], qf[m][k][3], kf[n >> 1][(n & 1) * 2], kf[n >> 1][(n & 1) * 2 + 1]);
                }
            }
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                float* dst = scores + (size_t)(kq * ROWS + m * 16 + (lane >> 2)) * LM_S_LD + kh * 32 + (lane & 3) * 2;
#pragma unroll
                for (int n = 0; n < 4; ++n) {
                    *reinterpret_cast<float2*>(dst + n * 8) = make_float2(sc[m][n][0], sc[m][n][1]);
                    *reinterpret_cast<float2*>(dst + 8 * LM_S_LD + n * 8) = make_float2(sc[m][n][2], sc[m][n][3]);
                }
            }
        }
        __syncthreads();
        {
            float v[KPT], mx = -INFINITY;
#pragma unroll
            for (int i = 0; i < KPT; i += 4) {
                const int k0 = i * TPR + sk0;
                float4 sum = make_float4(0, 0, 0, 0);
#pragma unroll
                for (int p = 0; p < 4; ++p) {
                    const float4 q4 = *reinterpret_cast<const float4*>(scores + (p * ROWS + srow) * LM_S_LD + k0);
                    sum.x += q4.x;
                    sum.y += q4.y;
                    sum.z += q4.z;
                    sum.w += q4.w;
                }
                const float e[4] = {sum.x, sum.y, sum.z, sum.w};
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int key = t * LM_KEYS + k0 + j;
                    v[i + j] = key <= limit && key < kv ? e[j] * sl2 : -INFINITY;
                    mx = fmaxf(mx, v[i + j]);
                }
            }
#pragma unroll
            for (int o = 1; o < TPR; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m_run, mx);
            const float keep = m_run == -INFINITY ? 0.0f : exp2_fast(m_run - mn);
            float sum = 0.0f;
#pragma unroll
            for (int i = 0; i < KPT; i += 4) {
                float p[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) p[j] = v[i + j] == -INFINITY ? 0.0f : exp2_fast(v[i + j] - mn);
                sum += (p[0] + p[1]) + (p[2] + p[3]);
                const uint32_t h0 = pack_bf16x2(p[0], p[1]), h1 = pack_bf16x2(p[2], p[3]);
                const size_t at = (size_t)srow * LM_P_LD + i * TPR + sk0;
                *reinterpret_cast<uint2*>(p_hi + at) = make_uint2(h0, h1);
                *reinterpret_cast<uint2*>(p_lo + at) = make_uint2(pack_bf16x2(p[0] - bf16_lo(h0), p[1] - bf16_hi(h0)), pack_bf16x2(p[2] - bf16_lo(h1), p[3] - bf16_hi(h1)));
            }
#pragma unroll
            for (int o = 1; o < TPR; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l_run = l_run * keep + sum;
            m_run = mn;
            if (sk0 == 0) corr[srow] = keep;
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float c0 = corr[m * 16 + (lane >> 2)], c1 = corr[m * 16 + (lane >> 2) + 8];
#pragma unroll
            for (int n = 0; n < NTW; ++n) {
                acc[m][n][0] *= c0;
                acc[m][n][1] *= c0;
                acc[m][n][2] *= c1;
                acc[m][n][3] *= c1;
            }
        }
#pragma unroll
        for (int k32 = 0; k32 < LM_KEYS / 32; ++k32) {
            uint32_t ph[MT][2][4], pl[MT][2][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const size_t at = (size_t)(m * 16 + (lm & 1) * 8 + lr) * LM_P_LD + k32 * 32 + h * 16 + (lm >> 1) * 8;
                    ldsm_x4(smem_u32(p_hi + at), ph[m][h]);
                    ldsm_x4(smem_u32(p_lo + at), pl[m][h]);
                }
#pragma unroll
            for (int n = 0; n < NTW; ++n) {
                const int col = (warp * NTW + n) * 8;
                if (col >= s.kv_rank) continue;                                      // (uniform over the warp)
                uint32_t vf[4];
                ldsm_x4_trans(smem_u32(K + (size_t)(k32 * 32 + lm * 8 + lr) * lay.ld + col), vf);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    mma_16816(acc[m][n], ph[m][0][0], ph[m][0][1], ph[m][0][2], ph[m][0][3], vf[0], vf[1]);
                    mma_16816(acc[m][n], ph[m][1][0], ph[m][1][1], ph[m][1][2], ph[m][1][3], vf[2], vf[3]);
                    mma_16816(acc[m][n], pl[m][0][0], pl[m][0][1], pl[m][0][2], pl[m][0][3], vf[0], vf[1]);
                    mma_16816(acc[m][n], pl[m][1][0], pl[m][1][1], pl[m][1][2], pl[m][1][3], vf[2], vf[3]);
                }
            }
        }
    }
    cp_async_wait_all();
    const size_t all_rows = (size_t)st.rows * s.heads, row_base = (size_t)first * s.heads + r0;
    if (sk0 == 0) {
        corr[ROWS + srow] = l_run;
        if (nsplit > 1 && srow < nrows) {
            part_ml[((size_t)split * all_rows + row_base + srow) * 2] = m_run;
            part_ml[((size_t)split * all_rows + row_base + srow) * 2 + 1] = l_run;
        }
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            const int row = m * 16 + hf * 8 + (lane >> 2);
            if (row >= nrows) continue;
            const float inv = 1.0f / corr[ROWS + row];
#pragma unroll
            for (int n = 0; n < NTW; ++n) {
                const int col = (warp * NTW + n) * 8 + (lane & 3) * 2;
                if (col >= s.kv_rank) continue;
                const float v0 = acc[m][n][hf * 2], v1 = acc[m][n][hf * 2 + 1];
                if (nsplit > 1) *reinterpret_cast<float2*>(part_o + ((size_t)split * all_rows + row_base + row) * s.kv_rank + col) = make_float2(v0, v1);
                else *reinterpret_cast<uint32_t*>(out + (row_base + row) * s.kv_rank + col) = pack_bf16x2(v0 * inv, v1 * inv);
            }
        }
}

// One CTA per row: the key shares' states into one.
__global__ void __launch_bounds__(128) latent_attention_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                                     int nsplit, long long all_rows, int kv_rank, bf16* __restrict__ out) {
    __shared__ float w[64];
    pdl_trigger();
    pdl_wait();
    const long long r = blockIdx.x;
    if (threadIdx.x < 32) {
        float m = -INFINITY, l = 0.0f;
        for (int k = threadIdx.x; k < nsplit; k += 32) m = fmaxf(m, part_ml[(k * all_rows + r) * 2]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        for (int k = threadIdx.x; k < nsplit; k += 32) {
            const float mk = part_ml[(k * all_rows + r) * 2], c = mk == -INFINITY ? 0.0f : exp2f(mk - m);
            w[k] = c;
            l += c * part_ml[(k * all_rows + r) * 2 + 1];
        }
        l = warp_sum(l);
        __syncwarp();
        for (int k = threadIdx.x; k < nsplit; k += 32) w[k] = l > 0.0f ? w[k] / l : 0.0f;
    }
    __syncthreads();
    for (int i = threadIdx.x * 2; i < kv_rank; i += 256) {
        float a = 0.0f, b = 0.0f;
#pragma unroll 16
        for (int k = 0; k < nsplit; ++k) {
            const float2 v = *reinterpret_cast<const float2*>(part_o + (k * all_rows + r) * kv_rank + i);
            a = fmaf(v.x, w[k], a);
            b = fmaf(v.y, w[k], b);
        }
        *reinterpret_cast<uint32_t*>(out + r * kv_rank + i) = pack_bf16x2(a, b);
    }
}

// The kernel variant of a shape, 0 = none.
int lm_ntw(const scr_latent_shape& s) {
    for (int n = 1; n <= 8; n *= 2)
        if (s.kv_rank <= 64 * n && s.kv_rank + s.rot_dim <= 64 * (n + 1)) return n;
    return 0;
}

// Two row tiles share a key tile's loads; one is quicker where even single key tiles would not fill the GPU.
int lm_mt(const scr_latent_shape& s, const scr_step& st, int sms) {
    const int rows = s.heads * st.max_count;
    return rows > 16 && (long long)scr_ceil_div(rows, 32) * st.batch * scr_ceil_div(st.max_kv, LM_KEYS) >= sms ? 2 : 1;
}

// Key shares: enough CTAs to fill the GPU, at least one tile each.
int lm_splits(const scr_latent_shape& s, const scr_step& st, int sms) {
    const int blocks = scr_ceil_div(s.heads * st.max_count, 16 * lm_mt(s, st, sms)) * st.batch, tiles = scr_ceil_div(st.max_kv, LM_KEYS);
    int n = std::max(1, sms / std::max(1, blocks));
    return std::min(std::min(n, tiles), 64);
}

template <int MT, int NTW>
cudaError_t lm_launch(const scr_latent_shape& s, const scr_step& st, const void* q, const void* cache, void* out, float* po, float* ml, int nsplit,
                      int* status, cudaStream_t stream) {
    const size_t smem = LmSmem::of(s.kv_rank + s.rot_dim, MT).total;
    const cudaError_t e = seq_smem(latent_attention_mma_kernel<MT, NTW>, smem);
    if (e != cudaSuccess) return e;
    return launch_pdl(latent_attention_mma_kernel<MT, NTW>, dim3(scr_ceil_div(s.heads * st.max_count, 16 * MT), nsplit, st.batch), dim3(LM_THREADS), smem,
                      stream, s, st, (const bf16*)q, (const bf16*)cache, (bf16*)out, po, ml, nsplit, status);
}

}  // namespace

bool latent_attention_mma_applies(const scr_latent_shape& s) {
    const int D = s.kv_rank + s.rot_dim;
    return s.kv_rank % 8 == 0 && D % 8 == 0 && lm_ntw(s) != 0 && LmSmem::of(D, 2).total <= 227 * 1024;
}

size_t latent_attention_mma_workspace(const scr_latent_shape& s, const scr_step& st, int sms) {
    const int n = lm_splits(s, st, sms);
    return n > 1 ? (size_t)n * st.rows * s.heads * (s.kv_rank + 2) * sizeof(float) : 0;
}

int32_t latent_attention_mma_launch(scr_ctx* ctx, const scr_latent_shape& s, const scr_step& st, const void* q, const void* cache, void* out,
                                    void* workspace, size_t workspace_bytes, cudaStream_t stream) {
    if (st.max_count <= 0 || st.max_kv <= 0 || st.batch <= 0) return scr_fail(ctx, SCR_E_SHAPE, "an empty step");
    if (!scr_aligned16(q) || !scr_aligned16(cache) || !scr_aligned16(out)) return scr_fail(ctx, SCR_E_ALIGN, "q, cache and out must be 16-byte aligned");
    const int n = lm_splits(s, st, ctx->sm_count), ntw = lm_ntw(s);
    if (n > 1 && (!workspace || workspace_bytes < latent_attention_mma_workspace(s, st, ctx->sm_count)))
        return scr_fail(ctx, SCR_E_WORKSPACE, "latent attention over %d key shares needs %zu bytes", n, latent_attention_mma_workspace(s, st, ctx->sm_count));
    float* po = (float*)workspace;
    float* ml = po ? po + (size_t)n * st.rows * s.heads * s.kv_rank : nullptr;
    const bool two = lm_mt(s, st, ctx->sm_count) == 2;
    cudaError_t e = cudaErrorInvalidValue;
#define LM_CASE(NTW)                                                                                                                     \
    case NTW:                                                                                                                            \
        e = two ? lm_launch<2, NTW>(s, st, q, cache, out, po, ml, n, ctx->dev_status, stream)                                            \
                : lm_launch<1, NTW>(s, st, q, cache, out, po, ml, n, ctx->dev_status, stream);                                           \
        break;
    switch (ntw) { LM_CASE(1) LM_CASE(2) LM_CASE(4) LM_CASE(8) }
#undef LM_CASE
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "latent_attention_mma: %s", cudaGetErrorString(e));
    int32_t rc = scr_check_launch(ctx, "latent_attention_mma");
    if (rc || n == 1) return rc;
    e = launch_pdl(latent_attention_merge_kernel, dim3(st.rows * s.heads), dim3(128), 0, stream, (const float*)po, (const float*)ml, n,
                   (long long)st.rows * s.heads, s.kv_rank, (bf16*)out);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "latent_attention_merge: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "latent_attention_merge");
}
