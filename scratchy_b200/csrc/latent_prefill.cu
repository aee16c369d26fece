#include "seq_common.cuh"
extern "C" int32_t scr_latent_prefill_supported(const scr_latent_shape*) { return 0; }
extern "C" int32_t scr_latent_prefill(scr_ctx*, const scr_latent_shape*, const void*, const void*, const void*, const void*, int64_t, const void*, int64_t, int32_t, int32_t, void*, int64_t, void*) { return SCR_E_UNSUPPORTED; }
