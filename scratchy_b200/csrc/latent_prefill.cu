// Causal attention for prompts over expanded latents, bf16, on tcgen05 tensor cores: per head the key of a token is its
// expanded part (own to the head) followed by its rotated part (shared by all heads), and the values come transposed, so
// that every operand is K-major.
//
// A CTA takes one head and 256 query rows as two tiles of 128 that run in turn: while the tensor core works on one tile,
// the softmax warps of the other work.  320 threads:
//   warp 0       TMA: the query tiles once, then key tiles (64 keys) and value tiles through two rings
//   warp 1       owns TMEM; one thread issues, per key tile and query tile, O += P V of the previous key tile and then
//                S = Q K^T of this one
//   warps 2-5, 6-9   softmax of tile 0, tile 1 (thread = query row): S from TMEM, f32 softmax, P back to TMEM as a bf16
//                head and remainder (two products: the weights keep about 16 bits), O rescaled in TMEM only when the
//                row maximum has grown by more than 2^8 over the reference the sums are kept in
// The end divides by the row sum and multiplies by the sigmoid of the output gate.
// TMEM per tile: S 64 columns, P 32 + 32, O 128.  Every wait is bounded (tc_common.cuh).
#include "seq_common.cuh"

#include <algorithm>

namespace {

constexpr int LF_THREADS = 320, LF_KEYS = 64, LF_MAX_CHUNKS = 4;
constexpr uint32_t LF_Q_CHUNK = 128 * 128, LF_K_CHUNK = LF_KEYS * 128;        // 64 dimensions of 128 query rows / 64 keys

struct LfLayout {
    int chunks, dim_chunks, vp, k_stages, v_stages;
    uint32_t k, v, bars, total;
    __host__ __device__ uint32_t k_bytes() const { return chunks * LF_K_CHUNK; }
    __host__ __device__ uint32_t v_bytes() const { return vp * 128; }
    static LfLayout of(const scr_latent_shape& s) {
        LfLayout l{};
        l.dim_chunks = (s.dim + 63) / 64;
        l.chunks = l.dim_chunks + (s.rot_dim + 63) / 64;
        l.vp = (s.vdim + 15) / 16 * 16;
        const uint32_t q = 2 * l.chunks * LF_Q_CHUNK, room = 226 * 1024 - 1024 - 256 - q;
        l.k_stages = l.v_stages = (int)std::min<uint32_t>(3, room / (l.k_bytes() + l.v_bytes()));
        l.k = q;
        l.v = l.k + l.k_stages * l.k_bytes();
        l.bars = l.v + l.v_stages * l.v_bytes();
        l.total = l.bars + 256 + 1024;
        return l;
    }
};

struct LfArgs {
    LfLayout lay;
    int rows, pos0, heads, vdim;
    float scale_log2;
    const bf16* gate;
    long long ld_gate;
    bf16* out;
    long long ld_out;
    int* status;
};

__global__ void __launch_bounds__(LF_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap qr_map, const __grid_constant__ CUtensorMap k_map,
                      const __grid_constant__ CUtensorMap kr_map, const __grid_constant__ CUtensorMap v_map, const LfArgs a) {
    extern __shared__ uint8_t smem_raw[];
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t* gen = smem_raw + (base - smem_u32(smem_raw));
    const LfLayout& L = a.lay;
    const uint32_t bars = base + L.bars;
    auto q_full = [&]() { return bars; };
    auto k_full = [&](int s) { return bars + 8u * (1 + s); };
    auto k_empty = [&](int s) { return bars + 8u * (4 + s); };
    auto v_full = [&](int s) { return bars + 8u * (7 + s); };
    auto v_empty = [&](int s) { return bars + 8u * (10 + s); };
    auto s_full = [&](int t) { return bars + 8u * (13 + t); };
    auto p_full = [&](int t) { return bars + 8u * (15 + t); };
    auto o_full = [&](int t) { return bars + 8u * (17 + t); };
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(gen + L.bars + 8 * 19);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.x, q0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * 256;      // the longest tiles first
    int n[2];                                                                          // key tiles of the two query tiles
#pragma unroll
    for (int t = 0; t < 2; ++t) {
        const int rows = min(128, a.rows - (q0 + t * 128));
        n[t] = rows > 0 ? (a.pos0 + q0 + t * 128 + rows + LF_KEYS - 1) / LF_KEYS : 0;
    }
    const int nmax = max(n[0], n[1]);

    pdl_trigger();
    if (threadIdx.x == 0) {
        mbar_init(q_full(), 1);
        for (int s = 0; s < 3; ++s) { mbar_init(k_full(s), 1); mbar_init(k_empty(s), 1); mbar_init(v_full(s), 1); mbar_init(v_empty(s), 1); }
        for (int t = 0; t < 2; ++t) { mbar_init(s_full(t), 1); mbar_init(p_full(t), 128); mbar_init(o_full(t), 1); }
        fence_mbar_init();
    }
    if (warp == 1) {
        tmem_alloc(smem_u32((const void*)tmem_slot), 512);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    auto s_col = [&](int t) { return tmem + 256u * t; };
    auto ph_col = [&](int t) { return tmem + 256u * t + 64u; };
    auto pl_col = [&](int t) { return tmem + 256u * t + 96u; };
    auto o_col = [&](int t) { return tmem + 256u * t + 128u; };
    pdl_wait();

    if (warp == 0) {
        if (lane == 0) {
            mbar_arrive_expect_tx(q_full(), 2 * L.chunks * LF_Q_CHUNK);
            for (int t = 0; t < 2; ++t)
                for (int c = 0; c < L.chunks; ++c) {
                    const bool rot = c >= L.dim_chunks;
                    tma_load_3d(base + (t * L.chunks + c) * LF_Q_CHUNK, rot ? &qr_map : &q_map, (rot ? c - L.dim_chunks : c) * 64, head, q0 + t * 128, q_full());
                }
            int ks = 0, vs = 0;
            uint32_t kp = 0, vp = 0;
            for (int j = 0; j < nmax; ++j) {
                mbar_wait(k_empty(ks), kp ^ 1u, a.status, TC_ERR_EMPTY_WAIT);
                mbar_arrive_expect_tx(k_full(ks), L.k_bytes());
                for (int c = 0; c < L.chunks; ++c) {
                    const bool rot = c >= L.dim_chunks;
                    tma_load_3d(base + L.k + ks * L.k_bytes() + c * LF_K_CHUNK, rot ? &kr_map : &k_map, (rot ? c - L.dim_chunks : c) * 64, rot ? 0 : head, j * LF_KEYS, k_full(ks));
                }
                if (++ks == L.k_stages) { ks = 0; kp ^= 1u; }
                mbar_wait(v_empty(vs), vp ^ 1u, a.status, TC_ERR_EMPTY_WAIT);
                mbar_arrive_expect_tx(v_full(vs), L.v_bytes());
                tma_load_3d(base + L.v + vs * L.v_bytes(), &v_map, j * LF_KEYS, 0, head, v_full(vs));
                if (++vs == L.v_stages) { vs = 0; vp ^= 1u; }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t s_desc = umma_idesc(1, 1, 128, LF_KEYS), o_desc = umma_idesc(1, 1, 128, (uint32_t)L.vp);
            mbar_wait(q_full(), 0, a.status, TC_ERR_FULL_WAIT);
            int ks = 0, vs = 0;
            uint32_t kp = 0, vp = 0;
            for (int j = 0; j <= nmax; ++j) {
                if (j < nmax) mbar_wait(k_full(ks), kp, a.status, TC_ERR_FULL_WAIT);
                if (j > 0) mbar_wait(v_full(vs), vp, a.status, TC_ERR_FULL_WAIT);
                tc_fence_after();
                for (int t = 0; t < 2; ++t) {
                    if (j > 0 && j <= n[t]) {                                        // O += P(j - 1) V(j - 1)
                        mbar_wait(p_full(t), (uint32_t)(j - 1) & 1u, a.status, TC_ERR_DEQ_WAIT);
                        tc_fence_after();
                        const uint64_t vd = umma_desc_k_sw128(base + L.v + vs * L.v_bytes());
#pragma unroll
                        for (int k4 = 0; k4 < 4; ++k4) umma_f16_ta(o_col(t), ph_col(t) + 8u * k4, vd + (uint64_t)(2 * k4), o_desc, (j > 1) || k4 > 0);
#pragma unroll
                        for (int k4 = 0; k4 < 4; ++k4) umma_f16_ta(o_col(t), pl_col(t) + 8u * k4, vd + (uint64_t)(2 * k4), o_desc, 1);
                        if (j == n[t]) umma_commit(o_full(t));
                    }
                    if (j < n[t]) {
                        for (int c = 0; c < L.chunks; ++c) {
                            const uint64_t qd = umma_desc_k_sw128(base + (t * L.chunks + c) * LF_Q_CHUNK);
                            const uint64_t kd = umma_desc_k_sw128(base + L.k + ks * L.k_bytes() + c * LF_K_CHUNK);
#pragma unroll
                            for (int k4 = 0; k4 < 4; ++k4) umma_f16(s_col(t), qd + (uint64_t)(2 * k4), kd + (uint64_t)(2 * k4), s_desc, (c | k4) != 0);
                        }
                        umma_commit(s_full(t));
                    }
                }
                if (j < nmax) {
                    umma_commit(k_empty(ks));
                    if (++ks == L.k_stages) { ks = 0; kp ^= 1u; }
                }
                if (j > 0) {
                    umma_commit(v_empty(vs));
                    if (++vs == L.v_stages) { vs = 0; vp ^= 1u; }
                }
            }
        }
    } else {
        const int t = warp >= 6, q = warp & 3;
        const uint32_t lanes = (uint32_t)(q * 32) << 16;
        const int row = q0 + t * 128 + q * 32 + lane, pos = a.pos0 + row;
        float m_ref = -INFINITY, l = 0.0f;
        for (int j = 0; j < n[t]; ++j) {
            mbar_wait(s_full(t), (uint32_t)j & 1u, a.status, TC_ERR_ACC_FULL);
            tc_fence_after();
            float v[64];
            {
                uint32_t r0[32], r1[32];
                tmem_ld_32x32(s_col(t) + lanes, r0);
                tmem_ld_32x32(s_col(t) + lanes + 32, r1);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    v[i] = __uint_as_float(r0[i]);
                    v[32 + i] = __uint_as_float(r1[i]);
                }
            }
            const int left = pos - j * LF_KEYS;                                      // keys 0..left of this tile are visible
            if (left < LF_KEYS - 1) {
#pragma unroll
                for (int i = 0; i < 64; ++i)
                    if (i > left) v[i] = -INFINITY;
            }
            float m4[4] = {v[0], v[1], v[2], v[3]};
#pragma unroll
            for (int i = 4; i < 64; ++i) m4[i & 3] = fmaxf(m4[i & 3], v[i]);
            const float mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])) * a.scale_log2;
            if (j == 0) {
                m_ref = mx;
            } else {
                const bool grow = mx > m_ref + 8.0f;
                if (__any_sync(0xffffffffu, grow)) {                                 // PV of the tiles before is complete (s_full)
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
                const float p0 = exp2_fast(fmaf(v[2 * i], a.scale_log2, -m_ref)), p1 = exp2_fast(fmaf(v[2 * i + 1], a.scale_log2, -m_ref));
                sum[i & 3] += p0 + p1;
                hi[i] = pack_bf16x2(p0, p1);
                lo[i] = pack_bf16x2(p0 - bf16_lo(hi[i]), p1 - bf16_hi(hi[i]));
            }
            l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
            tmem_st_32x32(ph_col(t) + lanes, hi);
            tmem_st_32x32(pl_col(t) + lanes, lo);
            tmem_st_wait();
            tc_fence_before();
            mbar_arrive(p_full(t));
        }
        if (n[t] > 0) {
            mbar_wait(o_full(t), 0, a.status, TC_ERR_ACC_FULL);
            tc_fence_after();
            const float inv = 1.0f / l;
            for (int c0 = 0; c0 < L.vp; c0 += 32) {
                uint32_t o[32];
                tmem_ld_32x32(o_col(t) + lanes + c0, o);
                tmem_ld_wait();
                if (row >= a.rows) continue;
                const bf16* g = a.gate + row * a.ld_gate + head * a.vdim + c0;
                bf16* dst = a.out + row * a.ld_out + head * a.vdim + c0;
#pragma unroll
                for (int i = 0; i < 32; i += 8) {                                     // (vdim is a multiple of 8)
                    if (c0 + i >= a.vdim) break;
                    const uint4 gv = *reinterpret_cast<const uint4*>(g + i);
                    const uint32_t gw[4] = {gv.x, gv.y, gv.z, gv.w};
                    uint32_t w[4];
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        w[k] = pack_bf16x2(__uint_as_float(o[i + 2 * k]) * inv * sigmoid_f32(bf16_lo(gw[k])),
                                           __uint_as_float(o[i + 2 * k + 1]) * inv * sigmoid_f32(bf16_hi(gw[k])));
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

bool lf_map(CUtensorMap* map, const void* base, uint64_t d0, uint64_t d1, uint64_t d2, uint64_t s1, uint64_t s2, uint32_t b1, uint32_t b2) {
    tc_encode_tiled_fn enc = tc_tensor_map_encoder();
    if (!enc) return false;
    const cuuint64_t dims[3] = {d0, d1, d2}, strides[2] = {s1, s2};
    const cuuint32_t box[3] = {64, b1, b2}, one[3] = {1, 1, 1};
    return enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE,
               CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace

extern "C" int32_t scr_latent_prefill_supported(const scr_latent_shape* s) {
    if (!s || s->heads <= 0 || s->dim <= 0 || s->rot_dim <= 0 || s->vdim <= 0 || s->kv_rank <= 0) return 0;
    if (!(s->scale > 0.0f)) return 0;                      // (the row maximum is taken before the scale)
    if (s->dim % 8 || s->rot_dim % 8 || s->vdim % 8 || s->vdim > 128 || s->kv_rank % 8 || s->heads * s->vdim <= 16) return 0;
    const LfLayout l = LfLayout::of(*s);
    return l.chunks <= LF_MAX_CHUNKS && l.k_stages >= 2;
}

extern "C" int32_t scr_latent_prefill(scr_ctx* ctx, const scr_latent_shape* s, const void* q, const void* k, const void* r, const void* v_t,
                                      int64_t ld_v, const void* gate, int64_t ld_gate, int32_t rows, int32_t pos0, void* out, int64_t ld_out,
                                      void* stream) {
    SCR_REQUIRE_CTX(ctx);
    if (!s || !q || !k || !r || !v_t || !gate || !out) return scr_fail(ctx, SCR_E_ARG, "null pointer");
    if (!scr_latent_prefill_supported(s)) return scr_fail(ctx, SCR_E_UNSUPPORTED, "latent prefill of this shape");
    if (rows <= 0 || pos0 < 0 || ld_v % 8 || ld_v < pos0 + rows || ld_gate % 8 || ld_out % 8) return scr_fail(ctx, SCR_E_SHAPE, "rows %d pos0 %d ld_v %lld", rows, pos0, (long long)ld_v);
    if (!scr_aligned16(q) || !scr_aligned16(k) || !scr_aligned16(r) || !scr_aligned16(v_t) || !scr_aligned16(gate) || !scr_aligned16(out))
        return scr_fail(ctx, SCR_E_ALIGN, "operands must be 16-byte aligned");
    const LfArgs a{LfLayout::of(*s), rows, pos0, s->heads, s->vdim, s->scale * 1.4426950408889634f, (const bf16*)gate, ld_gate, (bf16*)out, ld_out, ctx->dev_status};
    const uint64_t kv = (uint64_t)pos0 + rows, per = (uint64_t)(s->dim + s->rot_dim) * 2, H = s->heads;
    CUtensorMap qm, qrm, km, krm, vm;
    if (!lf_map(&qm, q, s->dim, H, rows, per, per * H, 1, 128) || !lf_map(&qrm, (const bf16*)q + s->dim, s->rot_dim, H, rows, per, per * H, 1, 128) ||
        !lf_map(&km, k, s->dim, H, kv, (uint64_t)s->dim * 2, (uint64_t)s->dim * 2 * H, 1, LF_KEYS) ||
        !lf_map(&krm, r, s->rot_dim, 1, kv, (uint64_t)s->rot_dim * 2, (uint64_t)s->rot_dim * 2, 1, LF_KEYS) ||
        !lf_map(&vm, v_t, kv, s->vdim, H, (uint64_t)ld_v * 2, (uint64_t)ld_v * 2 * s->vdim, a.lay.vp, 1))
        return scr_fail(ctx, SCR_E_CUDA, "latent_prefill: tensor map");
    cudaError_t e = seq_smem(latent_prefill_kernel, a.lay.total);
    if (e == cudaSuccess) e = launch_pdl(latent_prefill_kernel, dim3(s->heads, scr_ceil_div(rows, 256)), dim3(LF_THREADS), a.lay.total, (cudaStream_t)stream, qm, qrm, km, krm, vm, a);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "latent_prefill: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "latent_prefill");
}
