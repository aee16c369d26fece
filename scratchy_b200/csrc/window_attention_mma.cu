// Sliding-window attention for decoding and short portions, bf16, on mma.sync.  The rows that share a key/value head (the
// tokens of a portion times the heads of a group) come in tiles of 8; every warp walks key tiles of its own, 32 cache rows
// at a time, through a ring of its own (tiled TMA loads from the paged cache), with no barrier between the warps:
//   S = Q K^T with Q in registers; the keys' scale, bias, window; online softmax in f32 on the accumulators; O += P V from
//   the very same shared-memory rows, read transposed.
// The 8 rows fill half of an mma's 16: in P V the other half carries the remainders of the weights, P - bf16(P), so that
// one product keeps about 16 bits of them; the two halves of O are added at the end.
// The warps' states meet in shared memory; the key shares of a cluster's CTAs meet through distributed shared memory.
#include "window.cuh"

#include <algorithm>

namespace {

constexpr int WM_WARPS = 4, WM_THREADS = WM_WARPS * 32, WM_ROWS = 8, WM_KEYS = 32, WM_MAX_CLUSTER = 8;
constexpr uint32_t WM_CHUNK = WM_KEYS * 128;                 // 64 dimensions of a key tile

// NK: dimensions in steps of 16 (dim <= 16 * NK); STAGES: key tiles a warp keeps in flight
template <int NK, int STAGES>
struct WmSmem {
    static constexpr int kChunks = (NK * 16 + 63) / 64, kOLd = NK * 16 + 4;
    static constexpr uint32_t kTile = kChunks * WM_CHUNK, kRing = STAGES * kTile;                // per warp; the ring later holds its O
    static constexpr uint32_t kScale = WM_WARPS * kRing, kBars = kScale + WM_WARPS * STAGES * WM_KEYS * 4;
    static constexpr uint32_t kMl = kBars + WM_WARPS * STAGES * 8, kTotal = kMl + (WM_WARPS + 1) * WM_ROWS * 8 + 1024;
    static_assert(WM_ROWS * kOLd * 4 <= (int)kRing, "O fits a ring");
};

__device__ __forceinline__ float wm_peer(const float* p, uint32_t rank) {
    uint32_t at;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(at) : "r"(smem_u32(p)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(at) : "memory");
    return v;
}
__device__ __forceinline__ void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

struct WmArgs {
    scr_window_shape s;
    scr_step st;
    const bf16* q;
    const float* key_scale;
    const float* bias;
    const float* gate;
    long long ld_gate;
    bf16* out;
    long long ld_out;
    int splits;                                              // CTAs of a cluster, each with a share of the keys
    int* status;
};

template <int NK, int STAGES>
__global__ void __launch_bounds__(WM_THREADS) window_attention_mma_kernel(const __grid_constant__ CUtensorMap k_map, const __grid_constant__ WmArgs a) {
    extern __shared__ uint8_t wm_smem[];
    using SM = WmSmem<NK, STAGES>;
    constexpr int NO = NK * 2, OLD = SM::kOLd;               // 8-column tiles of O
    constexpr bool QREG = NK <= 8;
    const uint32_t base = (smem_u32(wm_smem) + 1023u) & ~1023u;
    uint8_t* gen = wm_smem + (base - smem_u32(wm_smem));
    const scr_window_shape& s = a.s;
    const int dim = s.dim, G = s.kv_heads, group = s.heads / G;
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, t4 = lane & 3, lm = lane >> 3, lr = lane & 7;
    const int split = blockIdx.x % a.splits, g = blockIdx.x / a.splits % G, tile = blockIdx.x / a.splits / G, b = blockIdx.y;
    const int first = a.st.segs[b * 4], count = a.st.segs[b * 4 + 1], pos0 = a.st.segs[b * 4 + 2];
    const int r0 = tile * WM_ROWS, nrows = min(WM_ROWS, count * group - r0);
    if (nrows <= 0 || first < 0 || first + count > a.st.rows) {          // (the whole cluster)
        pdl_wait();
        return;
    }
    const int p_lo = pos0 + r0 / group, p_hi = pos0 + (r0 + nrows - 1) / group;
    const WindowTiles tiles = window_tiles(s, p_lo, p_hi, WM_KEYS);
    const uint32_t ring = base + warp * SM::kRing, bars = base + SM::kBars + warp * STAGES * 8;
    float* scales = reinterpret_cast<float*>(gen + SM::kScale) + warp * STAGES * WM_KEYS;
    const int* table = a.st.block_table + (size_t)b * s.max_blocks;
    const int stride = a.splits * WM_WARPS, i0 = split * WM_WARPS + warp;
    // first cache row of this warp's tile number n, -1: no such tile
    auto look_up = [&](int n) -> int {
        const int i = i0 + n * stride;
        if (i >= tiles.count) return -1;
        const int key = tiles.tile(i) * WM_KEYS, blk = key / s.block_size;
        int block = blk < s.max_blocks ? table[blk] : -1;
        if (block < 0 || block >= s.num_blocks) {
            atomicCAS(a.status, 0, blk < s.max_blocks ? SEQ_BAD_BLOCK : SEQ_BAD_POSITION);
            block = 0;
        }
        return block * s.block_size + (key - blk * s.block_size);
    };
    auto load = [&](int stage, int row) {                    // lane 0
        if (row < 0) return;
        const uint32_t bar = bars + stage * 8;
        mbar_arrive_expect_tx(bar, SM::kTile + WM_KEYS * 4);
#pragma unroll
        for (int c = 0; c < SM::kChunks; ++c) tma_load_3d(ring + stage * SM::kTile + c * WM_CHUNK, &k_map, c * 64, g, row, bar);
        bulk_g2s(smem_u32(scales + stage * WM_KEYS), a.key_scale + row, WM_KEYS * 4, bar);
    };
    if (lane == 0) {
#pragma unroll
        for (int n = 0; n < STAGES; ++n) mbar_init(bars + n * 8, 1);
        fence_mbar_init();
    }
    pdl_wait();
    if (lane == 0) {
#pragma unroll
        for (int n = 0; n < STAGES; ++n) load(n, look_up(n));
    }
    __syncwarp();

    // this lane's row: gr of the tile
    const int row = r0 + min(gr, nrows - 1), tok = row / group, head = g * group + (row - tok * group), pos = pos0 + tok;
    const bf16* qp = a.q + ((size_t)(first + tok) * s.heads + head) * dim;
    const float* bias = a.bias + (size_t)head * (SCR_BIAS_LO + s.n_bias + SCR_BIAS_HI) + SCR_BIAS_LO;
    const float far = bias[s.n_bias - 1];
    auto q_at = [&](int c) { return c < dim ? *reinterpret_cast<const uint32_t*>(qp + c) : 0u; };
    uint32_t qf[QREG ? NK : 1][2];
    if (QREG)
#pragma unroll
        for (int ks = 0; ks < (QREG ? NK : 0); ++ks) {
            qf[ks][0] = q_at(ks * 16 + t4 * 2);
            qf[ks][1] = q_at(ks * 16 + 8 + t4 * 2);
        }
    float acc[NO][4] = {}, m = -1e30f, l = 0.0f;
    int stage = 0;
    uint32_t phase = 0;
    for (int n = 0; i0 + n * stride < tiles.count; ++n) {
        const int next = lane == 0 ? look_up(n + STAGES) : -1;
        mbar_wait(bars + stage * 8, phase, a.status, TC_ERR_FULL_WAIT);
        const uint32_t K = ring + stage * SM::kTile;
        const float* scale = scales + stage * WM_KEYS;
        const int key0 = tiles.tile(i0 + n * stride) * WM_KEYS;
        float sc[4][4] = {};
        {
            const uint32_t kb = K + ((lm >> 1) * 8 + lr) * 128;
#pragma unroll
            for (int ks = 0; ks < NK; ++ks) {
                uint32_t kf[2][4], q0, q1;
                const uint32_t at = kb + (ks >> 2) * WM_CHUNK + ((((ks & 3) * 2 + (lm & 1)) ^ lr) << 4);
                ldsm_x4(at, kf[0]);
                ldsm_x4(at + 16 * 128, kf[1]);
                if (QREG) {
                    q0 = qf[QREG ? ks : 0][0];
                    q1 = qf[QREG ? ks : 0][1];
                } else {
                    q0 = q_at(ks * 16 + t4 * 2);
                    q1 = q_at(ks * 16 + 8 + t4 * 2);
                }
#pragma unroll
                for (int x = 0; x < 4; ++x) mma_16816(sc[x], q0, 0u, q1, 0u, kf[x >> 1][(x & 1) * 2], kf[x >> 1][(x & 1) * 2 + 1]);
            }
        }
        float mx = m;
        {
            const bool beyond = p_lo - (key0 + WM_KEYS - 1) >= s.n_bias - 1;         // one bias for every distance of the tile
            const float* bt = bias + (pos - key0 - t4 * 2);
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float2 k2 = *reinterpret_cast<const float2*>(scale + x * 8 + t4 * 2);
                sc[x][0] = fmaf(sc[x][0], k2.x, beyond ? far : bt[-x * 8]);
                sc[x][1] = fmaf(sc[x][1], k2.y, beyond ? far : bt[-x * 8 - 1]);
            }
            if (key0 + WM_KEYS - 1 > p_lo || !(p_hi - key0 < s.window || key0 + WM_KEYS <= s.keep_first)) {       // not all visible to all rows
#pragma unroll
                for (int x = 0; x < 4; ++x)
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        if (!window_sees(s, pos, key0 + x * 8 + t4 * 2 + e)) sc[x][e] = -INFINITY;
            }
#pragma unroll
            for (int x = 0; x < 4; ++x) mx = fmaxf(mx, fmaxf(sc[x][0], sc[x][1]));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        }
        if (__any_sync(0xffffffffu, mx > m)) {
            const float c = exp2_fast(m - mx);
            l *= c;
            m = mx;
#pragma unroll
            for (int x = 0; x < NO; ++x) {
                acc[x][0] *= c;
                acc[x][1] *= c;
                acc[x][2] *= c;
                acc[x][3] *= c;
            }
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const float p0 = exp2_fast(sc[x][0] - m), p1 = exp2_fast(sc[x][1] - m);
            l += p0 + p1;
            ph[x] = pack_bf16x2(p0, p1);
            pl[x] = pack_bf16x2(p0 - bf16_lo(ph[x]), p1 - bf16_hi(ph[x]));
        }
        const uint32_t vb = K + (lm * 8 + lr) * 128;
#pragma unroll
        for (int x = 0; x < NO; ++x) {
            uint32_t vf[4];
            ldsm_x4_trans(vb + (x >> 3) * WM_CHUNK + (((x & 7) ^ lr) << 4), vf);
            mma_16816(acc[x], ph[0], pl[0], ph[1], pl[1], vf[0], vf[1]);
            mma_16816(acc[x], ph[2], pl[2], ph[3], pl[3], vf[2], vf[3]);
        }
        __syncwarp();                                        // every lane is done with the stage
        if (lane == 0) load(stage, next);
        if (++stage == STAGES) {
            stage = 0;
            phase ^= 1u;
        }
    }
    __syncwarp();
    // a warp's O and (m, l) per row; then the CTA's, then the cluster's
    float* O = reinterpret_cast<float*>(gen + warp * SM::kRing);
    float* ml = reinterpret_cast<float*>(gen + SM::kMl);     // [warp][row][2], then the CTA's [row][2]
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
#pragma unroll
    for (int x = 0; x < NO; ++x) *reinterpret_cast<float2*>(O + gr * OLD + x * 8 + t4 * 2) = make_float2(acc[x][0] + acc[x][2], acc[x][1] + acc[x][3]);
    if (t4 == 0) {
        ml[(warp * WM_ROWS + gr) * 2] = m;
        ml[(warp * WM_ROWS + gr) * 2 + 1] = l;
    }
    __syncthreads();
    float* all = ml + WM_WARPS * WM_ROWS * 2;
    if (threadIdx.x < WM_ROWS) {                             // one thread per row: the warps' weights, the CTA's sum
        float mm = -1e30f, ll = 0.0f;
        for (int w = 0; w < WM_WARPS; ++w) mm = fmaxf(mm, ml[(w * WM_ROWS + threadIdx.x) * 2]);
        for (int w = 0; w < WM_WARPS; ++w) {
            float* p = ml + (w * WM_ROWS + threadIdx.x) * 2;
            const float c = exp2_fast(p[0] - mm);
            ll += c * p[1];
            p[0] = c;
        }
        all[threadIdx.x * 2] = mm;
        all[threadIdx.x * 2 + 1] = ll;
    }
    __syncthreads();
    float* mine = reinterpret_cast<float*>(gen);             // the CTA's O, in the place of warp 0's
    for (int i = threadIdx.x; i < nrows * dim; i += WM_THREADS) {
        const int r = i / dim, c = i - r * dim;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < WM_WARPS; ++w) v = fmaf(reinterpret_cast<const float*>(gen + w * SM::kRing)[r * OLD + c], ml[(w * WM_ROWS + r) * 2], v);
        mine[r * OLD + c] = v;
    }
    if (a.splits > 1) cluster_sync();
    else __syncthreads();
    for (int i = split * WM_THREADS + threadIdx.x; i < nrows * dim; i += a.splits * WM_THREADS) {
        const int r = i / dim, c = i - r * dim, t = (r0 + r) / group, h = g * group + (r0 + r - t * group);
        float v, ll;
        if (a.splits == 1) {
            v = mine[r * OLD + c];
            ll = all[r * 2 + 1];
        } else {
            float pm[WM_MAX_CLUSTER], mm = -1e30f;
#pragma unroll
            for (int k = 0; k < WM_MAX_CLUSTER; ++k) {
                pm[k] = k < a.splits ? wm_peer(all + r * 2, k) : -1e30f;
                mm = fmaxf(mm, pm[k]);
            }
            v = ll = 0.0f;
#pragma unroll
            for (int k = 0; k < WM_MAX_CLUSTER; ++k)
                if (k < a.splits) {
                    const float w = exp2_fast(pm[k] - mm);
                    v = fmaf(w, wm_peer(mine + r * OLD + c, k), v);
                    ll = fmaf(w, wm_peer(all + r * 2 + 1, k), ll);
                }
        }
        const float f = sigmoid_f32(a.gate[(first + t) * a.ld_gate + h]) * s.out_scale / ll;
        a.out[(first + t) * a.ld_out + (size_t)h * dim + c] = __float2bfloat16_rn(v * f);
    }
    if (a.splits > 1) cluster_sync();                        // a CTA's shared memory stays until its peers have read it
}

template <int NK, int STAGES>
cudaError_t wm_launch(const CUtensorMap& map, const WmArgs& a, int tiles, cudaStream_t stream) {
    auto kernel = window_attention_mma_kernel<NK, STAGES>;
    const cudaError_t e = seq_smem(kernel, WmSmem<NK, STAGES>::kTotal);
    if (e != cudaSuccess) return e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.splits * a.s.kv_heads * tiles, a.st.batch);
    cfg.blockDim = dim3(WM_THREADS);
    cfg.dynamicSmemBytes = WmSmem<NK, STAGES>::kTotal;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = a.splits;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = a.splits > 1 ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, kernel, map, a);
}

}  // namespace

bool window_mma_applies(const scr_window_shape& s) { return s.dim % 8 == 0 && s.dim <= 256 && s.block_size % WM_KEYS == 0; }

int32_t window_mma_launch(scr_ctx* ctx, const scr_window_shape& s, const scr_step& st, const void* q, const void* cache, const float* key_scale,
                          const float* bias, const float* gate, int64_t ld_gate, void* out, int64_t ld_out, cudaStream_t stream) {
    WmArgs a{s, st, (const bf16*)q, key_scale, bias, gate, ld_gate, (bf16*)out, ld_out, 1, ctx->dev_status};
    if (st.max_kv <= 0 || st.batch > 65535) return scr_fail(ctx, SCR_E_SHAPE, "max_kv %d batch %d", st.max_kv, st.batch);
    CUtensorMap map;
    if (!window_map(&map, cache, s.dim, s.kv_heads, (uint64_t)s.num_blocks * s.block_size, WM_KEYS)) return scr_fail(ctx, SCR_E_CUDA, "window_attention_mma: tensor map");
    const int tiles = scr_ceil_div(st.max_count * (s.heads / s.kv_heads), WM_ROWS);
    // key shares: up to two CTAs per SM, at least one key tile per warp
    const long long seen = std::min<long long>(st.max_kv, (long long)s.window + s.keep_first + st.max_count);
    const long long ctas = (long long)tiles * s.kv_heads * st.batch, key_tiles = (seen + WM_KEYS - 1) / WM_KEYS;
    while (a.splits < WM_MAX_CLUSTER && ctas * a.splits <= ctx->sm_count && key_tiles >= 2ll * WM_WARPS * a.splits) a.splits *= 2;
    const cudaError_t e = s.dim <= 32 ? wm_launch<2, 3>(map, a, tiles, stream) : s.dim <= 64 ? wm_launch<4, 3>(map, a, tiles, stream)
                        : s.dim <= 128 ? wm_launch<8, 2>(map, a, tiles, stream) : wm_launch<16, 2>(map, a, tiles, stream);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "window_attention_mma: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "window_attention_mma");
}
