#include "seq_common.cuh"
bool latent_attention_mma_applies(const scr_latent_shape&) { return false; }
size_t latent_attention_mma_workspace(const scr_latent_shape&, const scr_step&, int) { return 0; }
int32_t latent_attention_mma_launch(scr_ctx*, const scr_latent_shape&, const scr_step&, const void*, const void*, void*, void*, size_t, cudaStream_t) { return SCR_E_UNSUPPORTED; }
