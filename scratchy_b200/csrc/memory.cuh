// Arguments of the matrix-memory kernels, and the gate arithmetic of the mLSTM.
#pragma once

#include "seq_common.cuh"

struct MemoryArgs {
    scr_mlstm_shape s;
    scr_step st;
    const void* proj;
    long long ld;
    float* gates;
    long long ld_gates;
    const float* bias_i;
    const float* bias_f;
    float* state_s;
    float* state_n;
    float* state_m;
    float* out;
    int* status;
    const float* powers;                                   // constant decay: [heads][SCR_DECAY_POWERS], otherwise unused
};

__host__ __device__ __forceinline__ int mlstm_slices(int vdim) { return (vdim + SCR_MLSTM_SLICE - 1) / SCR_MLSTM_SLICE; }

__device__ __forceinline__ float mlstm_cap(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float mlstm_gate_i(const MemoryArgs& a, int row, int h) {
    return mlstm_cap(a.gates[row * a.ld_gates + h] + a.bias_i[h], a.s.gate_cap);
}
__device__ __forceinline__ float mlstm_gate_f(const MemoryArgs& a, int row, int h) {
    const float z = mlstm_cap(a.gates[row * a.ld_gates + a.s.heads + h] + a.bias_f[h], a.s.gate_cap);
    return fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
}
