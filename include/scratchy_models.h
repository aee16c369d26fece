/*
 * scratchy_models.h — C ABI of the sequence-model kernels (sm_100a): full-precision linears, latent attention and
 * sliding-window attention over a paged cache, matrix memories with gates or with a constant decay, and the norms,
 * embedding and sampling around them.
 *
 * Built as `libscratchy_models.so`, which carries its own copy of the context functions of scratchy_cuda.h
 * (`scr_cuda_init`, `scr_device_status`, ...); a context belongs to the library that made it.  The conventions are
 * those of scratchy_cuda.h: plain pointers and sizes, an explicit stream, an `int32_t` status, no allocation.
 *
 * `dtype` is the type of weights, activations and cache of a call: SCR_DTYPE_BF16 (tensor-core kernels, f32
 * accumulation) or SCR_DTYPE_F32 (plain f32 arithmetic throughout, no reduced-precision matrix mode).  Residual
 * stream, norms, scores, softmax, gates and recurrent state are f32 under both.
 *
 * A step runs the tokens of one or more sequences, packed row after row.  Its description lives on the device:
 *   tok_seg [T]          the sequence (index into segs) each row belongs to
 *   tok_pos [T]          the row's position in its sequence
 *   segs [B][4]          per sequence: first row, number of rows, position of the first row, state slot
 *   block_table [B][max_blocks]   cache blocks of each sequence in order of position
 */
#ifndef SCRATCHY_MODELS_H_
#define SCRATCHY_MODELS_H_

#include "scratchy_cuda.h"

#ifdef __cplusplus
extern "C" {
#endif

#define SCR_DTYPE_F32 2

/* y = x W^T per group of rows, with the ends a layer folds around it.
 *   w   [groups * N, K] rows;  x row m of group g at x + m * ldx + g * x_group
 *   columns n < n_main go to y[m * ldy + g * y_group + n] (dtype, or f32 with y_f32), the others to the f32 buffer
 *   y2[m * ldy2 + n - n_main] (groups == 1)
 *   gate (may be NULL): the sum is multiplied by sigmoid(gate[m * ldg + g * y_group + n]) (dtype)
 *   act 1: rows of W hold, per 16, 8 gate rows then the 8 up rows of the same channels; y has N / 2 columns
 *          a sigmoid(alpha a) (b + 1),  a = min(gate, limit), b = clamp(up, -limit, limit)
 *   n_parts > 0: several linears over one x as one matrix.  Part p takes the columns from the end of part p - 1 to its n_end and
 *          writes them by its kind to its own y (row stride ld), column n - start of the part; y, y2, gate and act are unused
 *   residual (may be NULL): residual[m * ld_residual + n] += sum (f32); with tanh_w, y gets the norm of the new residual,
 *          tanh(tanh_alpha * residual) * tanh_w[n] + tanh_b[n] (dtype), otherwise y is unused
 * `workspace` (f32 slabs of a k-split) may be NULL when `scr_dense_workspace_size` reports 0. */
#define SCR_PART_STORE 0            /* dtype */
#define SCR_PART_F32 1              /* f32 */
#define SCR_PART_SILU 2             /* v sigmoid(v), dtype */
#define SCR_PART_GELU_GLU 3         /* rows in runs of 8 gate + 8 up as for act 1: gelu_tanh(gate) * up, half the columns, dtype */
#define SCR_DENSE_PARTS 6
typedef struct scr_dense_part {
    void* y;
    int64_t ld;
    int32_t n_end, kind;
} scr_dense_part;
typedef struct scr_dense {
    const void* w;
    const void* x;
    void* y;
    float* y2;
    const void* gate;
    int64_t ldx, x_group, ldy, y_group, ldy2, ldg;
    int32_t M, N, K, groups;
    int32_t n_main, y_f32, act;
    float limit, alpha;
    float* residual;
    int64_t ld_residual;
    const float* tanh_w;
    const float* tanh_b;
    float tanh_alpha;
    int32_t n_parts;
    scr_dense_part parts[SCR_DENSE_PARTS];
} scr_dense;
int32_t scr_dense_workspace_size(int32_t dtype, int32_t M, int32_t N, int32_t K, int32_t groups, size_t* bytes);
int32_t scr_dense_linear(scr_ctx* ctx, int32_t dtype, const scr_dense* d, void* workspace, size_t workspace_bytes,
                         void* stream);

/* x[i, :] = table[ids[i], :] as f32 (the residual stream); `raw` (may be NULL, dtype, row stride ld_raw) gets the row
 * as stored. */
int32_t scr_seq_embed(scr_ctx* ctx, int32_t dtype, const int32_t* ids, int32_t rows, const void* table, int32_t vocab,
                      int32_t width, float* x, void* raw, int64_t ld_raw, void* stream);

/* The step between two sublayers, on the f32 residual x [rows, width]; norm(v, w) = v / sqrt(mean(v^2) + eps) * (1 + w):
 *   delta, w_delta         x <- x + norm(delta, w_delta)      (delta f32 [rows, width])
 *   delta, no w_delta      x <- delta + bias                  (bias f32 [width] or NULL)
 *   no delta               x unchanged
 * then, with `out` (dtype, row stride ld_out): out <- norm(x, w_out), or the row itself when w_out is NULL; with b_out the
 * dynamic tanh instead, out <- tanh(alpha x) * w_out + b_out.
 * `row_index` (may be NULL): out row i is made from row row_index[i] of x (no delta then). */
typedef struct scr_seq_norm_args {
    float* x;
    const float* delta;
    const float* w_delta;
    const float* bias;
    const float* w_out;
    void* out;
    const int32_t* row_index;
    int64_t ld_out;
    int32_t rows, x_rows, width;
    float eps;
    const float* b_out;
    float alpha;
} scr_seq_norm_args;
int32_t scr_seq_norm(scr_ctx* ctx, int32_t dtype, const scr_seq_norm_args* a, void* stream);

/* Greedy token per row of f32 logits: the largest value, the smallest id among equals, NaN never. */
int32_t scr_seq_argmax(scr_ctx* ctx, const float* logits, int64_t ld, int32_t rows, int32_t width, int32_t* out,
                       void* stream);

/* ---- latent attention -------------------------------------------------------------------------
 * A cache row holds a token's latent (kv_rank values) and its rotated key part (rot_dim values), shared by all heads:
 * cache [num_blocks * block_size, kv_rank + rot_dim] of dtype. */
typedef struct scr_latent_shape {
    int32_t heads, dim, rot_dim, vdim, kv_rank, q_rank;
    int32_t rot_dims, max_pos;          /* rotated dimensions (interleaved pairs); rows of the cos / sin tables */
    int32_t block_size, num_blocks, max_blocks;
    float eps, scale;
} scr_latent_shape;
typedef struct scr_step {
    const int32_t* tok_seg;
    const int32_t* tok_pos;
    const int32_t* segs;
    const int32_t* block_table;
    int32_t rows, batch;
    int32_t max_count, max_kv;          /* upper bounds over the sequences: rows of one, keys seen by one */
    int32_t num_slots;                  /* state slots that exist */
} scr_step;
/* From the down projections `d` (f32, row stride ld_d: q_rank | kv_rank | rot_dim): c_q <- rms-normed query latent
 * (dtype [rows, q_rank]); the normed latent and the rotated key part go to the token's cache row. */
int32_t scr_latent_prepare(scr_ctx* ctx, int32_t dtype, const scr_latent_shape* s, const scr_step* st, const float* d,
                           int64_t ld_d, const float* wq_norm, const float* wkv_norm, const float* cos_table,
                           const float* sin_table, void* c_q, void* cache, void* stream);
/* Queries q (f32 [rows, heads * (dim + rot_dim)]): the unrotated part of head h of row t to
 * q_plain[t * ld_plain + h * head_plain], the rotated part to q_rot[t * ld_rot + h * head_rot] (both dtype). */
int32_t scr_latent_queries(scr_ctx* ctx, int32_t dtype, const scr_latent_shape* s, const scr_step* st, const float* q,
                           const float* cos_table, const float* sin_table, void* q_plain, int64_t ld_plain,
                           int64_t head_plain, void* q_rot, int64_t ld_rot, int64_t head_rot, void* stream);
/* Causal attention in the latent space over the paged cache (W_uk already applied to the queries, W_uv still to come):
 * q [rows, heads, kv_rank + rot_dim], out [rows, heads, kv_rank], both dtype.  `workspace`: partial states of a
 * key split, `scr_latent_attention_workspace` bytes. */
int32_t scr_latent_attention_workspace(int32_t dtype, const scr_latent_shape* s, const scr_step* st, size_t* bytes);
int32_t scr_latent_attention(scr_ctx* ctx, int32_t dtype, const scr_latent_shape* s, const scr_step* st, const void* q,
                             const void* cache, void* out, void* workspace, size_t workspace_bytes, void* stream);
/* The expanded form for prompts (bf16): keys and values of one sequence are materialised from its cache rows first.
 * `scr_latent_gather` copies the latents (c [kv, kv_rank]) and the rotated parts (r [kv, rot_dim]) of the first kv
 * tokens of sequence `seg` into dense rows; `scr_latent_prefill` attends with q [rows, heads, dim + rot_dim], k
 * [kv, heads * dim], r [kv, rot_dim], v transposed [heads * vdim, ld_v] and multiplies by sigmoid(gate) (row stride
 * ld_gate) before it stores out [rows, heads * vdim]: query row i is at position pos0 + i and sees keys 0..pos0 + i. */
int32_t scr_latent_prefill_supported(const scr_latent_shape* s);
int32_t scr_latent_gather(scr_ctx* ctx, const scr_latent_shape* s, const int32_t* block_table_row, int32_t kv,
                          const void* cache, void* c, void* r, void* stream);
int32_t scr_latent_prefill(scr_ctx* ctx, const scr_latent_shape* s, const void* q, const void* k, const void* r,
                           const void* v_t, int64_t ld_v, const void* gate, int64_t ld_gate, int32_t rows, int32_t pos0,
                           void* out, int64_t ld_out, void* stream);

/* ---- matrix-memory recurrence (mLSTM) -----------------------------------------------------------
 * proj (dtype, row stride ld): q [heads * dim] | k [heads * dim] | v [heads * vdim]; gates (f32, row stride ld_gates):
 * input gates [heads] | forget gates [heads], without their biases (a prompt's call leaves the log gates there).  State per slot, f32: S [heads, dim, vdim] and, for
 * every slice of SCR_MLSTM_SLICE value columns (slices = ceil(vdim / 32)) a copy of the normaliser and of the running
 * maximum, n [heads, slices, dim] and m [heads, slices] (the CTAs of a head then share nothing); a sequence whose rows start at position 0 starts from zero whatever the slot holds.
 * out f32 [rows, heads * vdim]: the readout of every token, before its norm. */
#define SCR_MLSTM_SLICE 32
typedef struct scr_mlstm_shape {
    int32_t heads, dim, vdim;
    float gate_cap, eps;
} scr_mlstm_shape;
/* `workspace`: states between the groups of a long prompt that is cut to fill the GPU. */
int32_t scr_mlstm_workspace(int32_t dtype, const scr_mlstm_shape* s, const scr_step* st, size_t* bytes);
int32_t scr_mlstm_run(scr_ctx* ctx, int32_t dtype, const scr_mlstm_shape* s, const scr_step* st, const void* proj,
                      int64_t ld, float* gates, int64_t ld_gates, const float* bias_i, const float* bias_f,
                      float* state_s, float* state_n, float* state_m, float* out, void* workspace,
                      size_t workspace_bytes, void* stream);
/* y[t, h, :] (dtype) = out / rms(out over the head) * norm * sigmoid(gate[t, h, :]) */
int32_t scr_mlstm_finish(scr_ctx* ctx, int32_t dtype, const scr_mlstm_shape* s, const float* out, const float* norm,
                         const void* gate, int64_t ld_gate, int32_t rows, void* y, void* stream);

/* ---- sliding-window attention whose values are its keys before their norm --------------------------
 * Grouped heads (query head h reads key/value head h / (heads / kv_heads)).  Queries and keys pass a causal convolution of
 * `taps` taps per channel and an RMS norm over the whole projection; the values are the convolved keys themselves.  The cache
 * therefore holds the values only, [num_blocks * block_size, kv_heads * dim] of dtype, and one f32 per token, key_scale =
 * scale * log2(e) / (root mean square of its keys); the key norm's weight is folded into the queries.
 * Position i sees j <= i with i - j < window or j < keep_first.  Score in powers of two: q.v * key_scale +
 * bias[h][min(i - j, n_bias - 1)], the bias of the softmax times log2(e).  A head's bias row has SCR_BIAS_LO copies of its first
 * entry before it and SCR_BIAS_HI copies of its last one behind it (a tile of keys then needs no limits). */
#define SCR_BIAS_LO 192
#define SCR_BIAS_HI 96
typedef struct scr_window_shape {
    int32_t heads, kv_heads, dim, taps;
    int32_t window, keep_first, n_bias;
    int32_t block_size, num_blocks, max_blocks;
    float eps, scale, out_scale;
} scr_window_shape;
/* proj (dtype, row stride ld): q [heads * dim] | k [kv_heads * dim] as projected; conv [taps, (heads + kv_heads) * dim] f32;
 * norm [heads * dim] f32, the query norm's weight times the key norm's of the head's keys.  conv_state (dtype) [num_slots, taps - 1, (heads + kv_heads) * dim] holds the last
 * projected rows of every sequence, oldest first; zeros precede position 0 whatever the slot holds.  Writes the queries
 * (dtype [rows, heads * dim], normed, times the key norm's weight), the cache rows, key_scale and conv_state. */
int32_t scr_window_prepare(scr_ctx* ctx, int32_t dtype, const scr_window_shape* s, const scr_step* st, const void* proj, int64_t ld,
                           const float* conv, const float* norm, void* conv_state, void* q, void* cache, float* key_scale,
                           void* stream);
/* out (dtype, row stride ld_out) [rows, heads * dim] = softmax(scores) v * sigmoid(gate[t * ld_gate + h]) * out_scale.
 * Blocks that no visible key lies in may be missing from the block table (any negative number). */
int32_t scr_window_attention(scr_ctx* ctx, int32_t dtype, const scr_window_shape* s, const scr_step* st, const void* q, const void* cache,
                             const float* key_scale, const float* bias, const float* gate, int64_t ld_gate, void* out, int64_t ld_out,
                             void* stream);

/* ---- matrix memory with a constant decay per head (lightning attention) -----------------------------
 * S <- decay_h S + k v^T, o = S^T q.  proj (dtype, row stride ld): q [heads * dim] | k [heads * dim] | v [heads * vdim];
 * powers f32 [heads][SCR_DECAY_POWERS]: decay_h^n for n = 0 .. 64, then what decay_h has beyond its f32 value.  State per
 * slot f32 [num_slots, heads, dim, vdim]; a sequence whose rows start at position 0 starts from zero whatever the slot
 * holds.  out f32 [rows, heads * vdim]. */
#define SCR_DECAY_POWERS 66
typedef struct scr_lightning_shape {
    int32_t heads, dim, vdim;
    float eps, out_scale;
} scr_lightning_shape;
int32_t scr_lightning_workspace(int32_t dtype, const scr_lightning_shape* s, const scr_step* st, size_t* bytes);
int32_t scr_lightning_run(scr_ctx* ctx, int32_t dtype, const scr_lightning_shape* s, const scr_step* st, const void* proj, int64_t ld,
                          const float* powers, float* state, float* out, void* workspace, size_t workspace_bytes, void* stream);
/* y[t, :] (dtype, row stride ld_y) = out / rms(out over all heads) * norm * sigmoid(gate[t, :]) * out_scale */
int32_t scr_lightning_finish(scr_ctx* ctx, int32_t dtype, const scr_lightning_shape* s, const float* out, const float* norm,
                             const void* gate, int64_t ld_gate, int32_t rows, void* y, int64_t ld_y, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* SCRATCHY_MODELS_H_ */
