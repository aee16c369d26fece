// Sliding-window attention for prompts, bf16, on tcgen05 tensor cores, straight from the paged cache: a key tile is one cache
// block of 64 tokens, loaded by TMA as the block table names it, and serves twice: K-major as the keys of S = Q K^T and
// MN-major as the values of O += P V (the values are the keys before their norm).
//
// A CTA takes one head and 256 query rows of one sequence as two tiles of 128 that run in turn: while the tensor core works
// on one tile, the softmax warps of the other work.  It walks the key tiles that any of its rows sees, those of the kept
// first tokens and those of the window; a query tile skips the ones none of its rows sees.  576 threads:
//   warp 0       TMA: the query tiles once, then key tiles with their scales through a ring
//   warp 1       owns TMEM; one of its threads issues, per key tile, S = Q K^T of both query tiles, then O += P V of the key tile before
//   warps 2-9, 10-17   softmax of tile 0, tile 1 (two threads per query row, half of the keys each; the row maxima meet in shared
//                memory): S from TMEM, scales, bias and window in f32, P in the place of S as a bf16 head and remainder (two products: the weights keep about 16 bits), O rescaled in TMEM
//                only when the row maximum has grown by more than 2^8 over the reference the sums are kept in
// TMEM per tile: two S of 64 columns (the next one is ready when the softmax of one is done), O 128.  Every wait is bounded
// (tc_common.cuh).
#include "window.cuh"

#include <algorithm>

namespace {

constexpr int WF_THREADS = 576, WF_KEYS = 64, WF_MAX_STAGES = 6, WF_BIAS = 4096;      // bias entries kept in shared memory
constexpr uint32_t WF_Q_CHUNK = 128 * 128, WF_K_CHUNK = WF_KEYS * 128;                // 64 dimensions of 128 query rows / 64 keys

struct WfLayout {
    int chunks, vp, stages, bias_n;
    uint32_t k, inv, bias, maxima, bars, total;
    __host__ __device__ uint32_t k_bytes() const { return chunks * WF_K_CHUNK; }
    static WfLayout of(const scr_window_shape& s) {
        WfLayout l{};
        l.chunks = (s.dim + 63) / 64;
        l.vp = (s.dim + 15) / 16 * 16;
        l.bias_n = s.n_bias <= WF_BIAS ? SCR_BIAS_LO + s.n_bias + SCR_BIAS_HI : 0;
        const uint32_t q = 2 * l.chunks * WF_Q_CHUNK, fixed = q + l.bias_n * 4 + 16 + 4096 + 256 + 1024;
        l.stages = (int)std::min<uint32_t>(WF_MAX_STAGES, (226 * 1024 - fixed) / (l.k_bytes() + WF_KEYS * 4));
        l.k = q;
        l.inv = l.k + l.stages * l.k_bytes();
        l.bias = l.inv + l.stages * WF_KEYS * 4;
        l.maxima = (l.bias + l.bias_n * 4 + 15) / 16 * 16;   // [parity][tile][half][row]
        l.bars = l.maxima + 4096;
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

// CHUNKS: 64-dimension chunks of a head
template <int CHUNKS>
__global__ void __launch_bounds__(WF_THREADS, 1)
window_prefill_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ WfArgs a) {
    extern __shared__ uint8_t smem_raw[];
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t* gen = smem_raw + (base - smem_u32(smem_raw));
    const WfLayout& L = a.lay;
    constexpr uint32_t K_BYTES = CHUNKS * WF_K_CHUNK;
    const scr_window_shape& s = a.s;
    const uint32_t bars = base + L.bars;
    auto q_full = [&]() { return bars; };
    auto k_full = [&](int i) { return bars + 8u * (1 + i); };
    auto k_empty = [&](int i) { return bars + 8u * (1 + WF_MAX_STAGES + i); };
    auto s_full = [&](int t, int i) { return bars + 8u * (1 + 2 * WF_MAX_STAGES + 2 * t + (i & 1)); };        // i: the tile's i-th S
    auto p_full = [&](int t, int i) { return bars + 8u * (5 + 2 * WF_MAX_STAGES + 2 * t + (i & 1)); };
    auto pv_done = [&](int t) { return bars + 8u * (9 + 2 * WF_MAX_STAGES + t); };
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(gen + L.bars + 8 * (11 + 2 * WF_MAX_STAGES));
    // (the broadcast lets the compiler see that a warp takes one way through the roles, and keep descriptors in uniform registers)
    const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
    const int head = blockIdx.x, q0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * 256, b = blockIdx.z;      // the longest first
    const int first = a.st.segs[b * 4], count = a.st.segs[b * 4 + 1], pos0 = a.st.segs[b * 4 + 2];

    pdl_trigger();
    if (q0 >= count || first < 0 || first + count > a.st.rows) {
        pdl_wait();
        return;
    }
    // the CTA's key tiles, and of those each query tile's: its kept ones and those from its own first one to its last
    struct Own {
        int first, last, kept;
        __device__ __forceinline__ bool has(int k) const { return k <= last && (k < kept || k >= first); }
    };
    auto own_tiles = [&](int t) {
        const int lo = q0 + t * 128, rows = min(128, count - lo);
        if (rows <= 0) return Own{-1, -1, 0};
        const WindowTiles w = window_tiles(s, pos0 + lo, pos0 + lo + rows - 1, WF_KEYS);
        return Own{w.first, (pos0 + lo + rows - 1) / WF_KEYS, w.kept};
    };
    const WindowTiles tiles = window_tiles(s, pos0 + q0, pos0 + min(q0 + 256, count) - 1, WF_KEYS);
    if (threadIdx.x == 0) {
        mbar_init(q_full(), 1);
        for (int i = 0; i < WF_MAX_STAGES; ++i) { mbar_init(k_full(i), 1); mbar_init(k_empty(i), 1); }
        for (int t = 0; t < 2; ++t) {
            for (int i = 0; i < 2; ++i) { mbar_init(s_full(t, i), 1); mbar_init(p_full(t, i), 8); }
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
            mbar_arrive_expect_tx(q_full(), 2 * CHUNKS * WF_Q_CHUNK);
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int c = 0; c < CHUNKS; ++c) tma_load_3d(base + (t * CHUNKS + c) * WF_Q_CHUNK, &q_map, c * 64, head, first + q0 + t * 128, q_full());
            const int g = head / (s.heads / s.kv_heads);
            const int* table = a.st.block_table + (size_t)b * s.max_blocks;
            int ks = 0;
            uint32_t kp = 0;
            auto look_up = [&](int j) {
                const int k = tiles.tile(j);
                int block = k < s.max_blocks ? table[k] : -1;
                if (block < 0 || block >= s.num_blocks) {
                    atomicCAS(a.status, 0, k < s.max_blocks ? SEQ_BAD_BLOCK : SEQ_BAD_POSITION);
                    block = 0;
                }
                return block;
            };
            int block = look_up(0);
            for (int j = 0; j < tiles.count; ++j) {
                const int next = j + 1 < tiles.count ? look_up(j + 1) : 0;           // (in flight while this tile waits for its stage)
                mbar_wait(k_empty(ks), kp ^ 1u, a.status, TC_ERR_EMPTY_WAIT);
                mbar_arrive_expect_tx(k_full(ks), K_BYTES + WF_KEYS * 4);
#pragma unroll
                for (int c = 0; c < CHUNKS; ++c) tma_load_3d(base + L.k + ks * K_BYTES + c * WF_K_CHUNK, &k_map, c * 64, g, block * WF_KEYS, k_full(ks));
                bulk_g2s(base + L.inv + ks * WF_KEYS * 4, a.key_scale + (size_t)block * WF_KEYS, WF_KEYS * 4, k_full(ks));
                block = next;
                if (++ks == L.stages) { ks = 0; kp ^= 1u; }
            }
        }
    } else if (warp == 1) {
        const bool issuer = elect_one();
        const uint32_t s_desc = umma_idesc(1, 1, 128, WF_KEYS), o_desc = umma_idesc(1, 1, 128, (uint32_t)L.vp) | UMMA_B_MN_MAJOR;
        const Own own[2] = {own_tiles(0), own_tiles(1)};
        uint64_t qd[2][CHUNKS];
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int c = 0; c < CHUNKS; ++c) qd[t][c] = umma_desc_k_sw128(base + (t * CHUNKS + c) * WF_Q_CHUNK);
        mbar_wait(q_full(), 0, a.status, TC_ERR_FULL_WAIT);
        int ks = 0, prev = 0, started[2] = {0, 0}, done[2] = {0, 0};             // S and P V issued for a query tile
        bool before[2] = {false, false};                                         // does it have the key tile before this one
        uint32_t kp = 0;
        for (int j = 0; j <= tiles.count; ++j) {
            const int k = j < tiles.count ? tiles.tile(j) : 0x7FFFFFFF;
            if (j < tiles.count) mbar_wait(k_full(ks), kp, a.status, TC_ERR_FULL_WAIT);
            tc_fence_after();
            bool has[2];
#pragma unroll
            for (int t = 0; t < 2; ++t) {                                            // (its S buffer: P V of two tiles before is issued)
                has[t] = own[t].has(k);
                if (!has[t]) continue;
                const uint32_t col = s_col(t, started[t]), full = s_full(t, started[t]);
                const uint64_t kd = umma_desc_k_sw128(base + L.k + ks * K_BYTES);
                if (issuer) {
#pragma unroll
                    for (int c = 0; c < CHUNKS; ++c)
#pragma unroll
                        for (int k4 = 0; k4 < 4; ++k4)
                            umma_f16(col, qd[t][c] + (uint64_t)(2 * k4), kd + (uint64_t)(c * (WF_K_CHUNK >> 4) + 2 * k4), s_desc, (c | k4) != 0);
                    umma_commit(full);
                }
                __syncwarp();
                ++started[t];
            }
            const uint64_t vd = umma_desc_mn_sw128(base + L.k + prev * K_BYTES, WF_K_CHUNK);
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                if (before[t]) {                                                     // O += P(j - 1) V(j - 1)
                    const int i = done[t]++;
                    mbar_wait(p_full(t, i), (uint32_t)(i >> 1) & 1u, a.status, TC_ERR_DEQ_WAIT);
                    tc_fence_after();
                    const uint32_t col = s_col(t, i), o = o_col(t), pv = pv_done(t);
                    if (issuer) {
#pragma unroll
                        for (int k4 = 0; k4 < 4; ++k4) umma_f16_ta(o, col + 8u * k4, vd + (uint64_t)(128 * k4), o_desc, i > 0 || k4 > 0);
#pragma unroll
                        for (int k4 = 0; k4 < 4; ++k4) umma_f16_ta(o, col + 32u + 8u * k4, vd + (uint64_t)(128 * k4), o_desc, 1);
                        umma_commit(pv);
                    }
                    __syncwarp();
                }
                before[t] = has[t];
            }
            if (j > 0 && issuer) umma_commit(k_empty(prev));                         // both products of the tile before are issued
            __syncwarp();
            prev = ks;
            if (++ks == L.stages) { ks = 0; kp ^= 1u; }
        }
    } else {
        const int t = warp >= 10, half = ((warp - 2) >> 2) & 1, q = warp & 3;        // half: keys 0..31 or 32..63 of a tile
        const uint32_t lanes = (uint32_t)(q * 32) << 16;
        const int row = q0 + t * 128 + q * 32 + lane, pos = pos0 + row, w_lo = pos - lane, w_hi = w_lo + 31;     // the warp's positions
        const float far = bias[s.n_bias - 1];
        const Own own = own_tiles(t);
        float* maxima = reinterpret_cast<float*>(gen + L.maxima) + t * 256 + q * 32 + lane;
        float m_ref = -1e30f, l = 0.0f;
        int seen = 0, ks = 0;
        uint32_t kp = 0;
        for (int j = 0; j < tiles.count; ++j) {
            const int k = tiles.tile(j);
            if (own.has(k)) {
                const int key0 = k * WF_KEYS + half * 32;
                mbar_wait(k_full(ks), kp, a.status, TC_ERR_FULL_WAIT);               // (long complete: the scales are read here too)
                mbar_wait(s_full(t, seen), (uint32_t)(seen >> 1) & 1u, a.status, TC_ERR_ACC_FULL);
                tc_fence_after();
                float v[32];
                {
                    uint32_t r[32];
                    tmem_ld_32x32(s_col(t, seen) + lanes + half * 32, r);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(r[i]);
                }
                const float4* inv = reinterpret_cast<const float4*>(gen + L.inv + ks * WF_KEYS * 4) + half * 8;
                if (w_lo - (key0 + 31) >= s.n_bias - 1) {                            // one bias for every distance here
#pragma unroll
                    for (int i = 0; i < 32; i += 4) {
                        const float4 iv = inv[i >> 2];
                        v[i] = fmaf(v[i], iv.x, far);
                        v[i + 1] = fmaf(v[i + 1], iv.y, far);
                        v[i + 2] = fmaf(v[i + 2], iv.z, far);
                        v[i + 3] = fmaf(v[i + 3], iv.w, far);
                    }
                } else {
                    const float* bt = bias + (pos - key0);
#pragma unroll
                    for (int i = 0; i < 32; i += 4) {
                        const float4 iv = inv[i >> 2];
                        v[i] = fmaf(v[i], iv.x, bt[-i]);
                        v[i + 1] = fmaf(v[i + 1], iv.y, bt[-i - 1]);
                        v[i + 2] = fmaf(v[i + 2], iv.z, bt[-i - 2]);
                        v[i + 3] = fmaf(v[i + 3], iv.w, bt[-i - 3]);
                    }
                }
                if (key0 + 31 > w_lo || !(w_hi - key0 < s.window || key0 + 32 <= s.keep_first)) {
                    // visible: keys up to the position itself, from the window's first one or below keep_first
                    const int last = pos - key0, start = pos - s.window + 1 - key0, keep = s.keep_first - key0;
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (i > last || (i < start && i >= keep)) v[i] = -INFINITY;
                }
                float m4[4] = {v[0], v[1], v[2], v[3]};
#pragma unroll
                for (int i = 4; i < 32; ++i) m4[i & 3] = fmaxf(m4[i & 3], v[i]);
                float mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
                float* mine = maxima + (seen & 1) * 512;
                mine[half * 128] = mx;
                // (both halves have S in registers from here on: P may take its place)
                asm volatile("bar.sync %0, 256;" ::"r"(1 + t) : "memory");
                mx = fmaxf(mx, mine[(half ^ 1) * 128]);
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
                        for (int c0 = half * 32; c0 < L.vp; c0 += 64) {              // the halves take 32 columns in turn
                            uint32_t o[32];
                            tmem_ld_32x32(o_col(t) + lanes + c0, o);
                            tmem_ld_wait();
#pragma unroll
                            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * c);
                            tmem_st_32x32(o_col(t) + lanes + c0, o);
                        }
                    }
                }
                uint32_t hi[16], lo[16];
                float sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float p0 = exp2_fast(v[2 * i] - m_ref), p1 = exp2_fast(v[2 * i + 1] - m_ref);
                    sum[i & 3] += p0 + p1;
                    hi[i] = pack_bf16x2(p0, p1);
                    lo[i] = pack_bf16x2(p0 - bf16_lo(hi[i]), p1 - bf16_hi(hi[i]));
                }
                l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
                tmem_st_32x16(s_col(t, seen) + lanes + half * 16, hi);
                tmem_st_32x16(s_col(t, seen) + lanes + 32 + half * 16, lo);
                tmem_st_wait();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(p_full(t, seen));         // one arrival per warp: they are taken one by one
                ++seen;
            }
            if (++ks == L.stages) { ks = 0; kp ^= 1u; }
        }
        if (seen > 0) {
            float* mine = maxima + (seen & 1) * 512;
            mine[half * 128] = l;
            asm volatile("bar.sync %0, 256;" ::"r"(1 + t) : "memory");
            l += mine[(half ^ 1) * 128];
            mbar_wait(pv_done(t), (uint32_t)(seen - 1) & 1u, a.status, TC_ERR_ACC_FULL);
            tc_fence_after();
            const float f = row < count ? sigmoid_f32(a.gate[(first + row) * a.ld_gate + head]) * s.out_scale / l : 0.0f;
            for (int c0 = half * 32; c0 < L.vp; c0 += 64) {
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
    auto kernel = a.lay.chunks == 1 ? window_prefill_kernel<1> : window_prefill_kernel<2>;
    cudaError_t e = seq_smem(kernel, a.lay.total);
    if (e == cudaSuccess)
        e = launch_pdl(kernel, dim3(s.heads, scr_ceil_div(st.max_count, 256), st.batch), dim3(WF_THREADS), a.lay.total, stream, qm, km, a);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "window_prefill: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "window_prefill");
}
