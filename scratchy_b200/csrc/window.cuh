// Which keys the sliding-window attention reads, shared by its kernels.
#pragma once

#include "seq_common.cuh"

// Key tiles of `unit` keys that query positions p_lo..p_hi see: the tiles of the kept first tokens, then those of the window,
// as one list of `count` tiles.
struct WindowTiles {
    int kept, first, count;
    __device__ __forceinline__ int tile(int i) const { return i < kept ? i : first + (i - kept); }
};
__device__ __forceinline__ WindowTiles window_tiles(const scr_window_shape& s, int p_lo, int p_hi, int unit) {
    WindowTiles w;
    w.kept = (min(s.keep_first, p_hi + 1) + unit - 1) / unit;
    w.first = max(w.kept, max(0, p_lo - s.window + 1) / unit);
    w.count = w.kept + max(0, p_hi / unit + 1 - w.first);
    return w;
}
__device__ __forceinline__ bool window_sees(const scr_window_shape& s, int pos, int key) {
    return key <= pos && (pos - key < s.window || key < s.keep_first);
}
// Cache row of position `pos` of sequence `seg`; -1 (and a status code) where it has none.
__device__ __forceinline__ long long window_row(const scr_window_shape& s, const int* block_table, int seg, int pos, int* status) {
    const int b = pos / s.block_size;
    if (pos < 0 || b >= s.max_blocks) {
        atomicCAS(status, 0, SEQ_BAD_POSITION);
        return -1;
    }
    const int block = block_table[(size_t)seg * s.max_blocks + b];
    if (block < 0 || block >= s.num_blocks) {
        atomicCAS(status, 0, SEQ_BAD_BLOCK);
        return -1;
    }
    return (long long)block * s.block_size + (pos - b * s.block_size);
}

// Rows of `heads` vectors of `dim` bf16 values: boxes of 64 dimensions of one head and `box_rows` rows, 128-byte swizzle, zeros outside.
static inline bool window_map(CUtensorMap* map, const void* base, uint64_t dim, uint64_t heads, uint64_t rows, uint32_t box_rows) {
    tc_encode_tiled_fn enc = tc_tensor_map_encoder();
    if (!enc) return false;
    const cuuint64_t dims[3] = {dim, heads, rows}, strides[2] = {dim * 2, dim * 2 * heads};
    const cuuint32_t box[3] = {64, 1, box_rows}, one[3] = {1, 1, 1};
    return enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE,
               CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
