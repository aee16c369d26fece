// Sliding-window attention for decoding and short portions, bf16, on mma.sync.  The rows that share a key/value head (the
// tokens of a portion times the heads of a group) are the 16 rows of a tile; every warp walks key tiles of its own, 32 cache
// rows at a time, through a ring of its own (cp.async), with no barrier between the warps:
//   S = Q K^T with Q in registers; the keys' scale, bias, window; online softmax in f32 on
//   the accumulators; P as a bf16 head and remainder (two products: the weights keep about 16 bits); O += P V from the very
//   same shared-memory rows, read transposed.
// The warps' states meet in shared memory; the key shares of a cluster's CTAs meet through distributed shared memory.
#include "window.cuh"

#include <algorithm>

namespace {

constexpr int WM_WARPS = 4, WM_THREADS = WM_WARPS * 32, WM_KEYS = 32, WM_MAX_CLUSTER = 8;

// NK: dimensions in steps of 16 (dim <= 16 * NK); STAGES: key tiles a warp keeps in flight
template <int NK, int STAGES>
struct WmSmem {
    static constexpr int kLd = NK * 16 + 8;                  // elements per key row: odd multiple of 16 bytes
    static constexpr int kTile = WM_KEYS * kLd * 2, kStage = kTile + WM_KEYS * 4, kWarp = STAGES * kStage;
    static constexpr int kO = 16 * (NK * 16 + 4) * 4;        // a warp's O, f32, over its ring
    static constexpr int kRing = kWarp > kO ? kWarp : kO;
    static constexpr int kTotal = WM_WARPS * kRing + (WM_WARPS + 1) * 16 * 2 * 4;
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
    const bf16* cache;
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
__global__ void __launch_bounds__(WM_THREADS) window_attention_mma_kernel(const WmArgs a) {
    extern __shared__ __align__(128) unsigned char wm_smem[];
    using SM = WmSmem<NK, STAGES>;
    constexpr int LD = SM::kLd, NO = NK * 2;                 // 8-column tiles of O
    constexpr bool QREG = NK <= 8;
    const scr_window_shape& s = a.s;
    const int dim = s.dim, G = s.kv_heads, group = s.heads / G;
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, t4 = lane & 3, lm = lane >> 3, lr = lane & 7;
    const int split = blockIdx.x % a.splits, g = blockIdx.x / a.splits % G, tile = blockIdx.x / a.splits / G, b = blockIdx.y;
    const int first = a.st.segs[b * 4], count = a.st.segs[b * 4 + 1], pos0 = a.st.segs[b * 4 + 2];
    const int r0 = tile * 16, nrows = min(16, count * group - r0);
    if (nrows <= 0 || first < 0 || first + count > a.st.rows) {          // (the whole cluster)
        pdl_wait();
        return;
    }
    const int p_lo = pos0 + r0 / group, p_hi = pos0 + (r0 + nrows - 1) / group;
    const WindowTiles tiles = window_tiles(s, p_lo, p_hi, WM_KEYS);
    unsigned char* ring = wm_smem + warp * SM::kRing;
    const int* table = a.st.block_table + (size_t)b * s.max_blocks;
    const int chunks = dim / 8, stride = a.splits * WM_WARPS, i0 = split * WM_WARPS + warp;
    const long long row_size = (long long)G * dim;
    // first cache row of this warp's tile number n, -1: no such tile
    auto look_up = [&](int n) -> long long {
        const int i = i0 + n * stride;
        if (i >= tiles.count) return -1;
        const int key = tiles.tile(i) * WM_KEYS, blk = key / s.block_size;
        const int block = blk < s.max_blocks ? table[blk] : -1;
        if (block < 0 || block >= s.num_blocks) {
            if (lane == 0) atomicCAS(a.status, 0, blk < s.max_blocks ? SEQ_BAD_BLOCK : SEQ_BAD_POSITION);
            return -1;
        }
        return (long long)block * s.block_size + (key - blk * s.block_size);
    };
    auto load = [&](int n, long long row) {
        if (row >= 0) {
            unsigned char* st = ring + (n % STAGES) * SM::kStage;
            const bf16* src = a.cache + row * row_size + (size_t)g * dim;
            const uint32_t dst = smem_u32(st);
#pragma unroll 4
            for (int c = lane; c < WM_KEYS * NK * 2; c += 32) {
                const int key = c / (NK * 2), x = c % (NK * 2);
                if (x < chunks) cp_async16(dst + (key * LD + x * 8) * 2, src + key * row_size + x * 8, true);
            }
            if (lane < WM_KEYS / 4) cp_async16(dst + SM::kTile + lane * 16, a.key_scale + row + lane * 4, true);
        }
        cp_async_commit();
    };
    // zero what the rows hold beyond dim (the last steps of 16 read it)
    if (dim < NK * 16)
        for (int i = lane; i < STAGES * WM_KEYS * (NK * 16 - dim); i += 32) {
            const int row = i / (NK * 16 - dim), c = dim + i % (NK * 16 - dim);
            reinterpret_cast<bf16*>(ring + row / WM_KEYS * SM::kStage)[(row % WM_KEYS) * LD + c] = __float2bfloat16_rn(0.0f);
        }
    pdl_wait();
#pragma unroll
    for (int n = 0; n < STAGES - 1; ++n) load(n, look_up(n));
    long long next = look_up(STAGES - 1);

    // this lane's two rows: gr and gr + 8 of the tile
    int head[2], pos[2];
    const bf16* qp[2];
    const float* bias[2];
    float far[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int r = r0 + min(gr + x * 8, nrows - 1), t = r / group;
        head[x] = g * group + (r - t * group);
        pos[x] = pos0 + t;
        qp[x] = a.q + ((size_t)(first + t) * s.heads + head[x]) * dim;
        bias[x] = a.bias + (size_t)head[x] * s.n_bias;
        far[x] = bias[x][s.n_bias - 1];
    }
    auto q_at = [&](int x, int c) { return c < dim ? *reinterpret_cast<const uint32_t*>(qp[x] + c) : 0u; };
    auto load_q = [&](int ks, uint32_t (&f)[4]) {
        f[0] = q_at(0, ks * 16 + t4 * 2);
        f[1] = q_at(1, ks * 16 + t4 * 2);
        f[2] = q_at(0, ks * 16 + 8 + t4 * 2);
        f[3] = q_at(1, ks * 16 + 8 + t4 * 2);
    };
    uint32_t qf[QREG ? NK : 1][4];
    if (QREG)
#pragma unroll
        for (int ks = 0; ks < (QREG ? NK : 0); ++ks) load_q(ks, qf[ks]);
    float acc[NO][4] = {}, m[2] = {-1e30f, -1e30f}, l[2] = {0.0f, 0.0f};
    for (int n = 0; i0 + n * stride < tiles.count; ++n) {
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
        __syncwarp();
        load(n + STAGES - 1, next);                          // (into the stage that the tile before has left)
        next = look_up(n + STAGES);
        const unsigned char* stg = ring + (n % STAGES) * SM::kStage;
        const bf16* K = reinterpret_cast<const bf16*>(stg);
        const float* inv = reinterpret_cast<const float*>(stg + SM::kTile);
        const int key0 = tiles.tile(i0 + n * stride) * WM_KEYS;
        float sc[4][4] = {};
        {
            const uint32_t kb = smem_u32(K + ((lm >> 1) * 8 + lr) * LD + (lm & 1) * 8);
#pragma unroll
            for (int ks = 0; ks < NK; ++ks) {
                uint32_t kf[2][4], f[4];
                ldsm_x4(kb + ks * 32, kf[0]);
                ldsm_x4(kb + ks * 32 + 16 * LD * 2, kf[1]);
                if (QREG) {
#pragma unroll
                    for (int j = 0; j < 4; ++j) f[j] = qf[QREG ? ks : 0][j];
                } else {
                    load_q(ks, f);
                }
#pragma unroll
                for (int x = 0; x < 4; ++x) mma_16816(sc[x], f[0], f[1], f[2], f[3], kf[x >> 1][(x & 1) * 2], kf[x >> 1][(x & 1) * 2 + 1]);
            }
        }
        const bool plain = key0 + WM_KEYS - 1 <= p_lo && (p_hi - key0 < s.window || key0 + WM_KEYS <= s.keep_first);   // all visible to all rows
        const bool beyond = p_lo - (key0 + WM_KEYS - 1) >= s.n_bias - 1;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int k = x * 8 + t4 * 2;
            const float2 iv = *reinterpret_cast<const float2*>(inv + k);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int hf = e >> 1, key = key0 + k + (e & 1), d = pos[hf] - key;
                const float bv = beyond ? far[hf] : bias[hf][min(max(d, 0), s.n_bias - 1)];
                float v = fmaf(sc[x][e], e & 1 ? iv.y : iv.x, bv);
                if (!plain && !window_sees(s, pos[hf], key)) v = -INFINITY;
                sc[x][e] = v;
                mx[hf] = fmaxf(mx[hf], v);
            }
        }
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            mx[hf] = fmaxf(mx[hf], __shfl_xor_sync(0xffffffffu, mx[hf], 1));
            mx[hf] = fmaxf(mx[hf], __shfl_xor_sync(0xffffffffu, mx[hf], 2));
            mx[hf] = fmaxf(mx[hf], m[hf]);
        }
        if (__any_sync(0xffffffffu, mx[0] > m[0] || mx[1] > m[1])) {
            const float c0 = exp2_fast(m[0] - mx[0]), c1 = exp2_fast(m[1] - mx[1]);
            l[0] *= c0;
            l[1] *= c1;
            m[0] = mx[0];
            m[1] = mx[1];
#pragma unroll
            for (int x = 0; x < NO; ++x) {
                acc[x][0] *= c0;
                acc[x][1] *= c0;
                acc[x][2] *= c1;
                acc[x][3] *= c1;
            }
        }
        uint32_t ph[2][4], pl[2][4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            float p[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) p[e] = exp2_fast(sc[x][e] - m[e >> 1]);
            l[0] += p[0] + p[1];
            l[1] += p[2] + p[3];
            const uint32_t h0 = pack_bf16x2(p[0], p[1]), h1 = pack_bf16x2(p[2], p[3]);
            ph[x >> 1][(x & 1) * 2] = h0;
            ph[x >> 1][(x & 1) * 2 + 1] = h1;
            pl[x >> 1][(x & 1) * 2] = pack_bf16x2(p[0] - bf16_lo(h0), p[1] - bf16_hi(h0));
            pl[x >> 1][(x & 1) * 2 + 1] = pack_bf16x2(p[2] - bf16_lo(h1), p[3] - bf16_hi(h1));
        }
        const uint32_t vb = smem_u32(K + (lm * 8 + lr) * LD);
#pragma unroll
        for (int x = 0; x < NO; ++x) {
            uint32_t vf[4];
            ldsm_x4_trans(vb + x * 16, vf);
            mma_16816(acc[x], ph[0][0], ph[0][1], ph[0][2], ph[0][3], vf[0], vf[1]);
            mma_16816(acc[x], ph[1][0], ph[1][1], ph[1][2], ph[1][3], vf[2], vf[3]);
            mma_16816(acc[x], pl[0][0], pl[0][1], pl[0][2], pl[0][3], vf[0], vf[1]);
            mma_16816(acc[x], pl[1][0], pl[1][1], pl[1][2], pl[1][3], vf[2], vf[3]);
        }
        __syncwarp();                                        // (the next load refills this stage's predecessor only)
    }
    cp_async_wait_all();
    __syncwarp();
    // a warp's O and (m, l) per row; then the CTA's, then the cluster's
    constexpr int OLD = NK * 16 + 4;
    float* O = reinterpret_cast<float*>(ring);
    float* ml = reinterpret_cast<float*>(wm_smem + WM_WARPS * SM::kRing);     // [warp][row][2], then the CTA's [row][2]
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        l[hf] += __shfl_xor_sync(0xffffffffu, l[hf], 1);
        l[hf] += __shfl_xor_sync(0xffffffffu, l[hf], 2);
        const int row = gr + hf * 8;
#pragma unroll
        for (int x = 0; x < NO; ++x) *reinterpret_cast<float2*>(O + row * OLD + x * 8 + t4 * 2) = make_float2(acc[x][hf * 2], acc[x][hf * 2 + 1]);
        if (t4 == 0) {
            ml[(warp * 16 + row) * 2] = m[hf];
            ml[(warp * 16 + row) * 2 + 1] = l[hf];
        }
    }
    __syncthreads();
    float* all = ml + WM_WARPS * 32;
    if (threadIdx.x < 16) {                                  // one thread per row: the warps' weights, the CTA's sum
        float mm = -1e30f, ll = 0.0f;
        for (int w = 0; w < WM_WARPS; ++w) mm = fmaxf(mm, ml[(w * 16 + threadIdx.x) * 2]);
        for (int w = 0; w < WM_WARPS; ++w) {
            float* p = ml + (w * 16 + threadIdx.x) * 2;
            const float c = exp2_fast(p[0] - mm);
            ll += c * p[1];
            p[0] = c;
        }
        all[threadIdx.x * 2] = mm;
        all[threadIdx.x * 2 + 1] = ll;
    }
    __syncthreads();
    float* mine = reinterpret_cast<float*>(wm_smem);         // the CTA's O, in the place of warp 0's
    for (int i = threadIdx.x; i < nrows * dim; i += WM_THREADS) {
        const int row = i / dim, c = i - row * dim;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < WM_WARPS; ++w) v = fmaf(reinterpret_cast<const float*>(wm_smem + w * SM::kRing)[row * OLD + c], ml[(w * 16 + row) * 2], v);
        mine[row * OLD + c] = v;
    }
    if (a.splits > 1) cluster_sync();
    else __syncthreads();
    for (int i = split * WM_THREADS + threadIdx.x; i < nrows * dim; i += a.splits * WM_THREADS) {
        const int row = i / dim, c = i - row * dim, r = r0 + row, t = r / group, h = g * group + (r - t * group);
        float v, ll;
        if (a.splits == 1) {
            v = mine[row * OLD + c];
            ll = all[row * 2 + 1];
        } else {
            float pm[WM_MAX_CLUSTER], mm = -1e30f;
#pragma unroll
            for (int k = 0; k < WM_MAX_CLUSTER; ++k) {
                pm[k] = k < a.splits ? wm_peer(all + row * 2, k) : -1e30f;
                mm = fmaxf(mm, pm[k]);
            }
            v = ll = 0.0f;
#pragma unroll
            for (int k = 0; k < WM_MAX_CLUSTER; ++k)
                if (k < a.splits) {
                    const float w = exp2_fast(pm[k] - mm);
                    v = fmaf(w, wm_peer(mine + row * OLD + c, k), v);
                    ll = fmaf(w, wm_peer(all + row * 2 + 1, k), ll);
                }
        }
        const float f = sigmoid_f32(a.gate[(first + t) * a.ld_gate + h]) * s.out_scale / ll;
        a.out[(first + t) * a.ld_out + (size_t)h * dim + c] = __float2bfloat16_rn(v * f);
    }
    if (a.splits > 1) cluster_sync();                        // a CTA's shared memory stays until its peers have read it
}

template <int NK, int STAGES>
cudaError_t wm_launch(const WmArgs& a, int tiles, cudaStream_t stream) {
    const cudaError_t e = seq_smem(window_attention_mma_kernel<NK, STAGES>, WmSmem<NK, STAGES>::kTotal);
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
    return cudaLaunchKernelEx(&cfg, window_attention_mma_kernel<NK, STAGES>, a);
}

}  // namespace

bool window_mma_applies(const scr_window_shape& s) { return s.dim % 8 == 0 && s.dim <= 256 && s.block_size % WM_KEYS == 0; }

int32_t window_mma_launch(scr_ctx* ctx, const scr_window_shape& s, const scr_step& st, const void* q, const void* cache, const float* key_scale,
                          const float* bias, const float* gate, int64_t ld_gate, void* out, int64_t ld_out, cudaStream_t stream) {
    WmArgs a{s, st, (const bf16*)q, (const bf16*)cache, key_scale, bias, gate, ld_gate, (bf16*)out, ld_out, 1, ctx->dev_status};
    if (st.max_kv <= 0 || st.batch > 65535) return scr_fail(ctx, SCR_E_SHAPE, "max_kv %d batch %d", st.max_kv, st.batch);
    const int tiles = scr_ceil_div(st.max_count * (s.heads / s.kv_heads), 16);
    // key shares: two CTAs per SM, at least two key tiles per warp
    const long long seen = std::min<long long>(st.max_kv, (long long)s.window + s.keep_first + st.max_count);
    const long long ctas = (long long)tiles * s.kv_heads * st.batch, key_tiles = (seen + WM_KEYS - 1) / WM_KEYS;
    while (a.splits < WM_MAX_CLUSTER && ctas * a.splits < 2ll * ctx->sm_count && key_tiles >= 2ll * WM_WARPS * a.splits) a.splits *= 2;
    const cudaError_t e = s.dim <= 32 ? wm_launch<2, 4>(a, tiles, stream) : s.dim <= 64 ? wm_launch<4, 4>(a, tiles, stream)
                        : s.dim <= 128 ? wm_launch<8, 3>(a, tiles, stream) : wm_launch<16, 2>(a, tiles, stream);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "window_attention_mma: %s", cudaGetErrorString(e));
    return scr_check_launch(ctx, "window_attention_mma");
}
