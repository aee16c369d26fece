// The mLSTM's prompts in chunks (memory_chunk.cuh), bf16.
#include "memory_chunk.cuh"

namespace {

// The log gates in place of the projections' sums: one thread per value.
__global__ void __launch_bounds__(256) mlstm_gates_kernel(MemoryArgs a) {
    pdl_trigger();
    pdl_wait();
    const int i = blockIdx.x * 256 + threadIdx.x, per = 2 * a.s.heads, row = i / per, c = i - row * per;
    if (row >= a.st.rows) return;
    a.gates[row * a.ld_gates + c] = c < a.s.heads ? mlstm_gate_i(a, row, c) : mlstm_gate_f(a, row, c - a.s.heads);
}

}  // namespace

bool mlstm_chunk_applies(const scr_mlstm_shape& s, const scr_step& st) { return ch_applies(s, st); }

size_t mlstm_chunk_workspace(const scr_mlstm_shape& s, const scr_step& st, int sms) { return ch_plan(s, st, sms).bytes; }

int32_t mlstm_chunk_launch(scr_ctx* ctx, const MemoryArgs& a, void* workspace, size_t workspace_bytes, cudaStream_t stream) {
    if (a.ld % 8 || !scr_aligned16(a.proj)) return scr_fail(ctx, SCR_E_ALIGN, "mlstm projections need 16-byte rows");
    const size_t need = ch_plan(a.s, a.st, ctx->sm_count).bytes;
    if (need > workspace_bytes || (need && !workspace)) return scr_fail(ctx, SCR_E_WORKSPACE, "mlstm needs %zu bytes", need);
    const cudaError_t e = launch_pdl(mlstm_gates_kernel, dim3(scr_ceil_div(a.st.rows * 2 * a.s.heads, 256)), dim3(256), 0, stream, a);
    if (e != cudaSuccess) return scr_fail(ctx, SCR_E_CUDA, "mlstm_gates: %s", cudaGetErrorString(e));
    const int32_t rc = scr_check_launch(ctx, "mlstm_gates");
    if (rc) return rc;
    return ch_run<false>(ctx, a, workspace, workspace_bytes, stream);
}
