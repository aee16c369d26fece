// Sliding-window attention for prompts, bf16, on tcgen05 tensor cores, straight from the paged cache: a key tile is one cache
// block of 64 tokens, loaded by TMA as the block table names it, and serves twice: K-major as the keys of S = Q K^T and
// MN-major as the values of O += P V (the values are the keys before their norm).
//
// A CTA takes one head and 256 query rows of one sequence as two tiles of 128 that run in turn: while the tensor core works
// on one tile, the softmax warps of the other work.  It walks the key tiles that any of its rows sees, those of the kept
// first tokens and those of the window; a query tile skips the ones none of its rows sees.  320 threads:
//   warp 0       TMA: the query tiles once, then key tiles with their scales through a ring
//   warp 1       owns TMEM; one thread issues, per key tile, S = Q K^T of both query tiles, then O += P V of the key tile before
//   warps 2-5, 6-9   softmax of tile 0, tile 1 (thread = query row): S from TMEM, scales, bias and window in f32, P in the place
//                of S as a bf16 head and remainder (two products: the weights keep about 16 bits), O rescaled in TMEM
//                only when the row maximum has grown by more than 2^8 over the reference the sums are kept in
// TMEM per tile: two S of 64 columns (the next one is ready when the softmax of one is done), O 128.  Every wait is bounded
// (tc_common.cuh).
#include "window.cuh"

#include <algorithm>

namespace {

constexpr int WF_THREADS = 320, WF_KEYS = 64, WF_MAX_STAGES = 6, WF_BIAS = 4096;      // bias entries kept in shared memory
constexpr uint32_t WF_Q_CHUNK = 128 * 128, WF_K_CHUNK = WF_KEYS * 128;                // 64 dimensions of 128 query rows / 64 keys

struct WfLayout {
    int chunks, vp, stages, bias_n;
    uint32_t k, inv, bias, bars, total;
    __host__ __device__ uint32_t k_bytes() const { return chunks * WF_K_CHUNK; }
    static WfLayout of(const scr_window_shape& s) {
        WfLayout l{};
        l.chunks = (s.dim + 63) / 64;
        l.vp = (s.dim + 15) / 16 * 16;
        l.bias_n = s.n_bias <= WF_BIAS ? SCR_BIAS_LO + s.n_bias + SCR_BIAS_HI : 0;
        const uint32_t q = 2 * l.chunks * WF_Q_CHUNK, fixed = q + l.bias_n * 4 + 16 + 256 + 1024;
        l.stages = (int)std::min<uint32_t>(WF_MAX_STAGES, (226 * 1024 - fixed) / (l.k_bytes() + WF_KEYS * 4));
        l.k = q;
        l.inv = l.k + l.stages * l.k_bytes();
        l.bias = l.inv + l.stages * WF_KEYS * 4;
        l.bars = (l.bias + l.bias_n * 4 + 15) / 16 * 16;
        l.total = l.bars + 256 + 1024;
        return l;
    }
};

struct WfArgs {
    WfLayout lay;
    scr_window_shape s;
    scr_step st;
    const float* key_scale;
    const float* bias;
    const float* gate;
    long long ld_gate;
    bf16* out;
    long long ld_out;
    int* status;
};

__global__ void __launch_bounds__(WF_THREADS, 1)
window_prefill_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ WfArgs a) {
    extern __shared__ uint8_t smem_raw[];
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t* gen = smem_raw + (base - smem_u32(smem_raw));
    const WfLayout& L = a.lay;
    const scr_window_shape& s = a.s;
    const uint32_t bars = base + L.bars;
    auto q_full = [&]() { return bars; };
    auto k_full = [&](int i) { return bars + 8u * (1 + i); };
    auto k_empty = [&](int i) { return bars + 8u * (1 + WF_MAX_STAGES + i); };
    auto s_full = [&](int t, int i) { return bars + 8u * (1 + 2 * WF_MAX_STAGES + 2 * t + (i & 1)); };        // i: the tile's i-th S
    auto p_full = [&](int t, int i) { return bars + 8u * (5 + 2 * WF_MAX_STAGES + 2 * t + (i & 1)); };
    auto pv_done = [&](int t) { return bars + 8u * (9 + 2 * WF_MAX_STAGES + t); };
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(gen + L.bars + 8 * (11 + 2 * WF_MAX_STAGES));
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.x, q0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * 256, b = blockIdx.z;      // the longest first
    const int first = a.st.segs[b * 4], count = a.st.segs[b * 4 + 1], pos0 = a.st.segs[b * 4 + 2];

    pdl_trigger();
    if (q0 >= count || first < 0 || first + count > a.st.rows) {
        pdl_wait();
        return;
    }
    // the CTA's key tiles, and of those each query tile's: its kept ones and those from its own first one to its last
    int own_first[2], own_last[2], own_kept[2];
#pragma unroll
    for (int t = 0; t < 2; ++t) {
        const int lo = q0 + t * 128, rows = min(128, count - lo);
        if (rows > 0) {
            const WindowTiles w = window_tiles(s, pos0 + lo, pos0 + lo + rows - 1, WF_KEYS);
            own_kept[t] = w.kept;
            own_first[t] = w.first;
            own_last[t] = (pos0 + lo + rows - 1) / WF_KEYS;
        } else {
            own_kept[t] = 0;
            own_first[t] = own_last[t] = -1;
        }
    }
    const WindowTiles tiles = window_tiles(s, pos0 + q0, pos0 + min(q0 + 256, count) - 1, WF_KEYS);
    auto active = [&](int t, int j) {
        if (j < 0 || j >= tiles.count) return false;
        const int k = tiles.tile(j);
        return k <= own_last[t] && (k < own_kept[t] || k >= own_first[t]);
    };
    if (threadIdx.x == 0) {
        mbar_init(q_full(), 1);
        for (int i = 0; i < WF_MAX_STAGES; ++i) { mbar_init(k_full(i), 1); mbar_init(k_empty(i), 1); }
        for (int t = 0; t < 2; ++t) {
            for (int i = 0; i < 2; ++i) { mbar_init(s_full(t, i), 1); mbar_init(p_full(t, i), 128); }
            mbar_init(pv_done(t), 1);
        }
        fence_mbar_init();
    }
    if (warp == 1) {
        tmem_alloc(smem_u32((const void*)tmem_slot), 512);
        tmem_relinquish();
    }
    const float* bias = a.bias + (size_t)head * (SCR_BIAS_LO + s.n_bias + SCR_BIAS_HI);
    if (L.bias_n) {                                          // (a constant of the model: no wait)
        float* dst = reinterpret_cast<float*>(gen + L.bias);
        for (int i = threadIdx.x; i < L.bias_n; i += WF_THREADS) dst[i] = bias[i];
        bias = dst;
    }
    bias += SCR_BIAS_LO;
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    auto s_col = [&](int t, int i) { return tmem + 256u * t + 64u * (i & 1); };        // S, then P: 32 columns of heads, 32 of remainders
    auto o_col = [&](int t) { return tmem + 256u * t + 128u; };
    pdl_wait();

    if (warp == 0) {
        if (lane == 0) {
            mbar_arrive_expect_tx(q_full(), 2 * L.chunks * WF_Q_CHUNK);
            for (int t = 0; t < 2; ++t)
                for (int c = 0; c < L.chunks; ++c) tma_load_3d(base + (t * L.chunks + c) * WF_Q_CHUNK, &q_map, c * 64, head, first + q0 + t * 128, q_full());
            const int g = head / (s.heads / s.kv_heads);
            const int* table = a.st.block_table + (size_t)b * s.max_blocks;
            int ks = 0;
            uint32_t kp = 0;
            for (int j = 0; j < tiles.count; ++j) {
                const int k = tiles.tile(j);
                int block = k < s.max_blocks ? table[k] : -1;
                if (block < 0 || block >= s.num_blocks) {
                    atomicCAS(a.status, 0, k < s.max_blocks ? SEQ_BAD_BLOCK : SEQ_BAD_POSITION);
                    block = 0;
                }
                mbar_wait(k_empty(ks), kp ^ 1u, a.status, TC_ERR_EMPTY_WAIT);
                mbar_arrive_expect_tx(k_full(ks), L.k_bytes() + WF_KEYS * 4);
                for (int c = 0; c < L.chunks; ++c) tma_load_3d(base + L.k + ks * L.k_bytes() + c * WF_K_CHUNK, &k_map, c * 64, g, block * WF_KEYS, k_full(ks));
                bulk_g2s(base + L.inv + ks * WF_KEYS * 4, a.key_scale + (size_t)block * WF_KEYS, WF_KEYS * 4, k_full(ks));
                if (++ks == L.stages) { ks = 0; kp ^= 1u; }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t s_desc = umma_idesc(1, 1, 128, WF_KEYS), o_desc = umma_idesc(1, 1, 128, (uint32_t)L.vp) | UMMA_B_MN_MAJOR;
            mbar_wait(q_full(), 0, a.status, TC_ERR_FULL_WAIT);
            int ks = 0, prev = 0, started[2] = {0, 0}, done[2] = {0, 0};             // S and P V issued for a query tile
            uint32_t kp = 0;
            for (int j = 0; j <= tiles.count; ++j) {
                if (j < tiles.count) mbar_wait(k_full(ks), kp, a.status, TC_ERR_FULL_WAIT);
                tc_fence_after();
                for (int t = 0; t < 2; ++t) {                                        // (its S buffer: P V of two tiles before is issued)
                    if (!active(t, j)) continue;
                    for (int c = 0; c < L.chunks; ++c) {
                        const uint64_t qd = umma_desc_k_sw128(base + (t * L.chunks + c) * WF_Q_CHUNK);
                        const uint64_t kd = umma_desc_k_sw128(base + L.k + ks * L.k_bytes() + c * WF_K_CHUNK);
#pragma unroll
                        for (int k4 = 0; k4 < 4; ++k4) umma_f16(s_col(t, started[t]), qd + (uint64_t)(2 * k4), kd + (uint64_t)(2 * k4), s_desc, (c | k4) != 0);
                    }
                    umma_commit(s_full(t, started[t]));
                    ++started[t];
                }
                for (int t = 0; t < 2; ++t) {
                    if (!active(t, j - 1)) continue;                                 // O += P(j - 1) V(j - 1)
                    const int i = done[t]++;
                    mbar_wait(p_full(t, i), (uint32_t)(i >> 1) & 1u, a.status, TC_ERR_DEQ_WAIT);
                    tc_fence_after();
                    const uint64_t vd = umma_desc_mn_sw128(base + L.k + prev * L.k_bytes(), WF_K_CHUNK);
#pragma unroll
                    for (int k4 = 0; k4 < 4; ++k4) umma_f16_ta(o_col(t), s_col(t, i) + 8u * k4, vd + (uint64_t)(128 * k4), o_desc, i > 0 || k4 > 0);
#pragma unroll
                    for (int k4 = 0; k4 < 4; ++k4) umma_f16_ta(o_col(t), s_col(t, i) + 32u + 8u * k4, vd + (uint64_t)(128 * k4), o_desc, 1);
                    umma_commit(pv_done(t));
                }
                if (j > 0) umma_commit(k_empty(prev));                               // both products of the tile before are issued
                prev = ks;
                if (++ks == L.stages) { ks = 0; kp ^= 1u; }
            }
        }
    } else {
        const int t = warp >= 6, q = warp & 3;
        const uint32_t lanes = (uint32_t)(q * 32) << 16;
        const int row = q0 + t * 128 + q * 32 + lane, pos = pos0 + row, w_lo = pos - lane, w_hi = w_lo + 31;     // the warp's positions
        const float far = bias[s.n_bias - 1];
        float m_ref = -1e30f, l = 0.0f;
        int seen = 0, ks = 0;
        uint32_t kp = 0;
        for (int j = 0; j < tiles.count; ++j) {
            if (active(t, j)) {
                const int key0 = tiles.tile(j) * WF_KEYS;
                mbar_wait(k_full(ks), kp, a.status, TC_ERR_FULL_WAIT);               // (long complete: the scales are read here too)
                mbar_wait(s_full(t, seen), (uint32_t)(seen >> 1) & 1u, a.status, TC_ERR_ACC_FULL);
                tc_fence_after();
                float v[64];
                {
                    uint32_t r0[32], r1[32];
                    tmem_ld_32x32(s_col(t, seen) + lanes, r0);
                    tmem_ld_32x32(s_col(t, seen) + lanes + 32, r1);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        v[i] = __uint_as_float(r0[i]);
                        v[32 + i] = __uint_as_float(r1[i]);
                    }
                }
                const float4* inv = reinterpret_cast<const float4*>(gen + L.inv + ks * WF_KEYS * 4);
                if (w_lo - (key0 + WF_KEYS - 1) >= s.n_bias - 1) {                   // one bias for every distance of the tile
#pragma unroll
                    for (int i = 0; i < 64; i += 4) {
                        const float4 iv = inv[i >> 2];
                        v[i] = fmaf(v[i], iv.x, far);
                        v[i + 1] = fmaf(v[i + 1], iv.y, far);
                        v[i + 2] = fmaf(v[i + 2], iv.z, far);
                        v[i + 3] = fmaf(v[i + 3], iv.w, far);
                    }
                } else {
                    const float* bt = bias + (pos - key0);
#pragma unroll
                    for (int i = 0; i < 64; i += 4) {
                        const float4 iv = inv[i >> 2];
                        v[i] = fmaf(v[i], iv.x, bt[-i]);
                        v[i + 1] = fmaf(v[i + 1], iv.y, bt[-i - 1]);
                        v[i + 2] = fmaf(v[i + 2], iv.z, bt[-i - 2]);
                        v[i + 3] = fmaf(v[i + 3], iv.w, bt[-i - 3]);
                    }
                }
                if (key0 + WF_KEYS - 1 > w_lo || !(w_hi - key0 < s.window || key0 + WF_KEYS <= s.keep_first)) {
                    // visible: keys up to the position itself, from the window's first one or below keep_first
                    const int last = pos - key0, start = pos - s.window + 1 - key0, keep = s.keep_first - key0;
#pragma unroll
                    for (int i = 0; i < 64; ++i)
                        if (i > last || (i < start && i >= keep)) v[i] = -INFINITY;
                }
                float m4[4] = {v[0], v[1], v[2], v[3]};
#pragma unroll
                for (int i = 4; i < 64; ++i) m4[i & 3] = fmaxf(m4[i & 3], v[i]);
                const float mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
                if (seen == 0) {
                    m_ref = fmaxf(m_ref, mx);
                } else {
                    const bool grow = mx > m_ref + 8.0f;
                    if (__any_sync(0xffffffffu, grow)) {
                        mbar_wait(pv_done(t), (uint32_t)(seen - 1) & 1u, a.status, TC_ERR_ACC_FULL);
                        tc_fence_after();
                        const float c = grow ? exp2_fast(m_ref - mx) : 1.0f;
                        if (grow) m_ref = mx;
                        l *= c;
                        for (int c0 = 0; c0 < L.vp; c0 += 32) {
                            uint32_t o[32];
                            tmem_ld_32x32(o_col(t) + lanes + c0, o);
                            tmem_ld_wait();
#pragma unroll
                            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * c);
                            tmem_st_32x32(o_col(t) + lanes + c0, o);
                        }
                    }
                }
                uint32_t hi[32], lo[32];
                float sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    const float p0 = exp2_fast(v[2 * i] - m_ref), p1 = exp2_fast(v[2 * i + 1] - m_ref);
                    sum[i & 3] += p0 + p1;
                    hi[i] = pack_bf16x2(p0, p1);
                    lo[i] = pack_bf16x2(p0 - bf16_lo(hi[i]), p1 - bf16_hi(hi[i]));
                }
                l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
                tmem_st_32x32(s_col(t, seen) + lanes, hi);
                tmem_st_32x32(s_col(t, seen) + lanes + 32, lo);
                tmem_st_wait();
                tc_fence_before();
                mbar_arrive(p_full(t, seen));
                ++seen;
            }
            if (++ks == L.stages) { ks = 0; kp ^= 1u; }
        }
        if (seen > 0) {
            mbar_wait(pv_done(t), (uint32_t)(seen - 1) & 1u, a.status, TC_ERR_ACC_FULL);
            tc_fence_after();
            const float f = row < count ? sigmoid_f32(a.gate[(first + row) * a.ld_gate + head]) * s.out_scale / l : 0.0f;
            for (int c0 = 0; c0 < L.vp; c0 += 32) {
                uint32_t o[32];
                tmem_ld_32x32(o_col(t) + lanes + c0, o);
                tmem_ld_wait();
                if (row >= count) continue;
                bf16* dst = a.out + (first + row) * a.ld_out + (size_t)head * s.dim + c0;
#pragma unroll
                for (int i = 0; i < 32; i += 8) {                                    // (dim is a multiple of 8)
                    if (c0 + i >= s.dim) break;
                    uint32_t w[4];
#pragma unroll
                    for (int k = 0; k < 4; ++k) w[k] = pack_bf16x2(__uint_as_float(o[i + 2 * k]) * f, __uint_as_float(o[i + 2 * k + 1]) * f);
                    *reinterpret_cast<uint4*>(dst + i) = make_uint4(w[0], w[1], w[2], w[3]);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem, 512);
    }
}

constexpr int WF_MIN_ROWS = 64;                              // rows of one sequence from which the prompt kernel pays

}  // namespace

bool window_prefill_applies(const scr_window_shape& s, const scr_step& st) {
    return st.max_count >= WF_MIN_ROWS && s.block_size == WF_KEYS && s.dim % 8 == 0 && s.dim <= 128 && st.batch <= 65535 && WfLayout::of(s).stages >= 3;
}

int32_t window_prefill_launch(scr_ctx* ctx, const scr_window_shape& s, const scr_step& st, const void* q, const void* cache, const float* key_scale,
                              const float* bias, const float* gate, int64_t ld_gate, void* out, int64_t ld_out, cudaStream_t stream) {
    const WfArgs a{WfLayout::of(s), s, st, key_scale, bias, gate, ld_gate, (bf16*)out, ld_out, ctx->dev_status};
    CUtensorMap qm, km;
    if (!window_map(&qm, q, s.dim, s.heads, st.rows, 128) || !window_map(&km, cache, s.dim, s.kv_heads, (uint64_t)s.num_blocks * s.block_size, WF_KEYS))
        return scr_fail(ctx, SCR_E_CUDA, "window_prefill: tensor map");
    cudaError_t e = seq_smem(window_prefill_kernel, a.lay.total);
    if (e == cudaSuccess)
        e = launch_pdl(window_prefill_kernel, dim3(s.heads, scr_ceil_div(st.max_count, 256), st.batch), dim3(WF_THREADS), a.lay.total, stream, qm, km, a);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "window_prefill: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "window_prefill");
}
