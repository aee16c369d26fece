#include "mlstm.cuh"
bool mlstm_chunk_applies(const scr_mlstm_shape&, const scr_step&) { return false; }
int32_t mlstm_chunk_launch(scr_ctx* ctx, const MlstmArgs&, cudaStream_t) { return SCR_E_UNSUPPORTED; }
