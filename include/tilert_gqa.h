/*
 * tilert_gqa -- C ABI of the grouped-query attention / mixture-of-experts path with bf16 weights: decoders whose
 * layers are q/k-normalised windowed attention with mixed values and clamped gated experts.
 *
 * These are mechanisms, not a model: every size and constant is an argument.  Conventions are those of
 * tilert_b200.h: device pointers, caller-allocated outputs, asynchronous on `stream`, 0 or a negative TB_E* code,
 * bounded waits that end in the context's status word.
 *
 * Numbers.  Weights are bf16.  Activations of a portion of tokens (`void*` operands) are bf16, or f32 when `f32` is
 * set: then every product is true 32-bit arithmetic.  The residual stream, norms, router, attention scores and
 * weights and the vectors of a one-token step are f32 in both modes.
 *
 * Padding.  A row of weights or activations has a stride that is a multiple of 8 elements; elements between the
 * logical length and the next multiple of 8 are zero.  f32 vectors of the one-token step are padded the same way.
 * Cache rows and prepared queries are padded to 16.
 *
 * Cache.  Keys [kv_heads, ring, dimp], values [kv_heads, ring, vdimp]; position p is row p % ring.
 */
#ifndef TILERT_GQA_H_
#define TILERT_GQA_H_

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#ifndef TB_OK
#define TB_OK 0
#define TB_ECUDA (-1)
#define TB_EINVAL (-2)
#define TB_ESTATE (-3)
#endif

typedef struct TgContext TgContext;

/* ---- runtime ---- */
int tilert_gqa_default_context(int device, TgContext** ctx_out);
int tilert_gqa_status(TgContext* ctx, int* status_out);
const char* tilert_gqa_last_error(void);
long long tilert_gqa_launch_count(void);
int tilert_gqa_set_wait_budget(TgContext* ctx, long long cycles);
int tilert_gqa_num_sms(TgContext* ctx);

/* ---- norms on the residual stream ---- */

/* x[t] = rms(table[tokens[t]]) * gain, also stored as activations in xh (may be NULL).  A token outside [0, vocab)
 * is refused on the device (status 4). */
int tilert_gqa_embed_norm_op(TgContext* ctx, const long long* tokens, const void* table, long long ld_table, int vocab,
                             const float* gain, float eps, int rows, int dim, float* x, long long ldx, void* xh,
                             long long ldh, int f32, void* stream);
/* x[t] += rms(y[t]) * gain, xh = x.  y is f32 [rows, ldy]; with y NULL the sublayer output is
 * sum_j slot_w[t, j] ye[slot_row[t, j]] (+ ysh[t] when given), the combine of a mixture of experts. */
int tilert_gqa_residual_norm_op(TgContext* ctx, const float* y, long long ldy, const void* ye, long long lde,
                                const int* slot_row, const float* slot_w, int top, const void* ysh, long long ldsh,
                                const float* gain, float eps, int rows, int dim, float* x, long long ldx, void* xh,
                                long long ldh, int f32, void* stream);
/* out[i] = rms(x[rows[i]]) * gain */
int tilert_gqa_gather_norm_op(TgContext* ctx, const float* x, long long ldx, const int* rows, int n, const float* gain,
                              float eps, int dim, void* out, long long ldo, int f32, void* stream);

/* ---- products of a portion of tokens ---- */

/* out[t, :] = W x[t] (+ bias), W [n, ldw]; tensor cores (tcgen05) on bf16 rows, SIMT f32 otherwise.
 * out_f32: f32 output also from bf16 rows.  gated: W holds n gate rows, then n up rows, and
 * out = g / (1 + exp(-alpha g)) * (u + 1) with g = min(gate, limit), u = up within +-limit.
 * n_groups > 0: W is [n_groups][n or 2 n][ldw], counts[g] (device) rows of x and out belong to group g, in order. */
int tilert_gqa_gemm_op(TgContext* ctx, const void* x, long long ldx, int rows, const void* w, long long ldw, int n, int k,
                       int gated, float limit, float alpha, int n_groups, const int* counts, const float* bias, void* out,
                       long long ldo, int out_f32, int f32, void* stream);

/* ---- attention of a portion of tokens ---- */

/* From qkv [rows, ld] f32 (queries | keys | values): queries and keys RMS-normalised over their whole projection
 * times their gains, values mixed (v_mode 0: as they are; 1: stored to v_first [rows, kv_heads * vdim]; 2:
 * (1 - *lambda) v + *lambda v_first).  Queries to q [rows, heads, dimp], keys and values to cache rows
 * (*pos + t) % ring. */
int tilert_gqa_qkv_rows_op(TgContext* ctx, const float* qkv, long long ld, const float* q_gain, const float* k_gain,
                           float eps, int v_mode, const float* lambda, float* v_first, int rows, int heads, int kv_heads,
                           int dim, int vdim, const int* pos, void* q, void* k_cache, void* v_cache, int ring, int f32,
                           void* stream);
/* out[t, h] = softmax over the visible cached keys; query t is at *pos + t, window 0 = no window.
 * window + rows - 1 must not exceed ring (window 0: *pos + rows). */
int tilert_gqa_attn_rows_op(TgContext* ctx, const void* q, const void* k_cache, const void* v_cache, int rows, int heads,
                            int kv_heads, int dim, int vdim, const int* pos, int window, int ring, float scale, void* out,
                            long long ldo, int f32, void* stream);

/* ---- routing of a portion of tokens ---- */

/* The `top` largest of logits [rows, ldl] per row, softmax over them; counts [n_experts] is cleared and counted. */
int tilert_gqa_route_rows_op(TgContext* ctx, const float* logits, long long ldl, int rows, int n_experts, int top, int* ids,
                             float* w, int* rank, int* counts, void* stream);
/* Rows of x repeated in expert order; slot_row[t, j] says where row t's j-th copy went. */
int tilert_gqa_gather_rows_op(TgContext* ctx, const void* x, long long ldx, int rows, int dim, int n_experts, int top,
                              const int* ids, const int* rank, const int* counts, void* xs, int* slot_row, int f32,
                              void* stream);

/* ---- one-token step ---- */

/* v = x, or x + rms(y) * gain when y is given (stored to x_out when not NULL), or the norm of that with gain2;
 * out = W v (+ bias). */
int tilert_gqa_vec_dense_op(TgContext* ctx, const float* x, const float* y, const float* gain, const float* gain2, float eps,
                            float* x_out, const void* w, long long ldw, const float* bias, int n, int k, float* out,
                            void* stream);
/* qkv_rows_op and attn_rows_op of one token at *pos in one launch.  n_splits CTAs share the keys of a head block; part
 * holds heads * n_splits * (vdimp + 2) floats, counter one zero word per head block.  out [heads * vdim] f32. */
int tilert_gqa_vec_attn_op(TgContext* ctx, const float* qkv, const float* q_gain, const float* k_gain, float eps, int v_mode,
                           const float* lambda, float* v_first, int heads, int kv_heads, int dim, int vdim, const int* pos,
                           int window, int ring, float scale, void* k_cache, void* v_cache, int n_splits, float* part,
                           int* counter, float* out, int f32, void* stream);
/* Head blocks (kv_heads x blocks of query heads) of a one-token attention launch. */
int tilert_gqa_head_blocks(int heads, int kv_heads);
/* Routing from logits [n_experts] and the gated halves of the shared and the selected experts:
 * hidden [pad8(ff_sh) + top * pad8(ff)].  w [n_experts][2][ff][ldw], w_sh [2][ff_sh][ldw] or NULL. */
int tilert_gqa_vec_gate_up_op(TgContext* ctx, const float* x, int dim, const float* logits, int n_experts, int top,
                              const void* w, const void* w_sh, long long ldw, int ff, int ff_sh, float limit, float limit_sh,
                              float alpha, float* hidden, int* slot_ids, float* slot_w, void* stream);
/* out = sum of slot_w * W_down[slot] hidden[slot], plus the shared expert.  w [n_experts][dim][pad8(ff)],
 * w_sh [dim][pad8(ff_sh)] or NULL. */
int tilert_gqa_vec_down_op(TgContext* ctx, const float* hidden, const int* slot_ids, const float* slot_w, int top,
                           const void* w, const void* w_sh, int ff, int ff_sh, int dim, float* out, void* stream);

/* tilert_sample_op of tilert_b200.h (same kernel, same arguments). */
int tilert_gqa_sample_op(TgContext* ctx, const float* logits, long long logits_stride, int tokens, int vocab,
                         const float* config_dev, unsigned long long seed, unsigned long long* step_dev,
                         unsigned long long step_value, int* token_out, float* token_logprob_out, float* topn_logprob_out,
                         int* topn_index_out, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* TILERT_GQA_H_ */
