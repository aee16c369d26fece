// Prompts of the matrix memory with a constant decay in chunks (memory_chunk.cuh), bf16.
#include "memory_chunk.cuh"

bool lightning_chunk_applies(const scr_mlstm_shape& s, const scr_step& st) { return ch_applies(s, st); }

size_t lightning_chunk_workspace(const scr_mlstm_shape& s, const scr_step& st, int sms) { return ch_plan(s, st, sms).bytes; }

int32_t lightning_chunk_launch(scr_ctx* ctx, const MemoryArgs& a, void* workspace, size_t workspace_bytes, cudaStream_t stream) {
    return ch_run<true>(ctx, a, workspace, workspace_bytes, stream);
}
