/*
 * tilert_gqa -- C ABI of decoders with bf16 weights: q/k-normalised windowed attention with mixed values or attention
 * over a latent cache (windows, sinks, output gates), clamped gated units, dense or routed, RMS or layer norms.
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
 * Cache.  Keys [kv_heads, ring, dimp], values [kv_heads, ring, vdimp], or latent rows [ring, row] (see below); position
 * p is row p % ring.
 *
 * Norms.  RMS norm, or the layer norm (mean taken off) where `centered` is set.  Biases of norms may be NULL.
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

/* x[t] = rms(table[tokens[t]]) * gain (gain NULL: the row as it is), also stored as activations in xh (may be NULL).  A
 * token outside [0, vocab) is refused on the device (status 4). */
int tilert_gqa_embed_norm_op(TgContext* ctx, const long long* tokens, const void* table, long long ld_table, int vocab,
                             const float* gain, float eps, int rows, int dim, float* x, long long ldx, void* xh,
                             long long ldh, int f32, void* stream);
/* x[t] += norm(y[t]) (+ add), then xh = x, or its norm with gain2 (xh may be NULL without gain2).  y is f32 [rows, ldy];
 * with y NULL and ye given the sublayer output is sum_j slot_w[t, j] ye[slot_row[t, j]] (+ ysh[t] when given), the
 * combine of a mixture of experts; with both NULL (and gain NULL) there is none. */
int tilert_gqa_residual_norm_op(TgContext* ctx, const float* y, long long ldy, const void* ye, long long lde,
                                const int* slot_row, const float* slot_w, int top, const void* ysh, long long ldsh,
                                const float* gain, const float* bias, const float* add, const float* gain2,
                                const float* bias2, int centered, float eps, int rows, int dim, float* x, long long ldx,
                                void* xh, long long ldh, int f32, void* stream);
/* out[i] = norm(x[rows[i]]) */
int tilert_gqa_gather_norm_op(TgContext* ctx, const float* x, long long ldx, const int* rows, int n, const float* gain,
                              const float* bias, int centered, float eps, int dim, void* out, long long ldo, int f32,
                              void* stream);

/* ---- products of a portion of tokens ---- */

/* out[t, :] = W x[t] (+ bias), W [n, ldw]; tensor cores (tcgen05) on bf16 rows, SIMT f32 otherwise.
 * out_f32: f32 output also from bf16 rows.  gated: W holds n gate rows, then n up rows, and
 * out = g / (1 + exp(-alpha g)) * (u + 1) with g = min(gate, limit), u = up within +-limit.
 * n_groups > 0: W is [n_groups][n or 2 n][ldw], counts[g] (device) rows of x and out belong to group g, in order; with
 * counts NULL every group has `rows` of them. */
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

/* v = x, or x + norm(y) when y is given, plus `add` when given (stored to x_out when not NULL), or the norm of that with
 * gain2; out = W v (+ bias). */
int tilert_gqa_vec_dense_op(TgContext* ctx, const float* x, const float* y, const float* gain, const float* norm_bias,
                            const float* add, const float* gain2, const float* norm_bias2, int centered, float eps,
                            float* x_out, const void* w, long long ldw, const float* bias, int n, int k, float* out,
                            void* stream);
/* The same input into W [2][n][ldw] (gate rows, then up rows): out[n] as in gemm_op with `gated`. */
int tilert_gqa_vec_gated_op(TgContext* ctx, const float* x, const float* y, const float* gain, const float* norm_bias,
                            const float* add, const float* gain2, const float* norm_bias2, int centered, float eps,
                            float* x_out, const void* w, long long ldw, int n, int k, float limit, float alpha, float* out,
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

/* ---- attention over a latent cache ---- */

/* A cache row is [latent (rank), zero to rankp = pad16(rank) | rotated key part (rot), zero to row], row =
 * pad32(rankp + rot); keys and values of all heads are linear in the latent, the rotated part is one for all heads.
 * Projected queries hold per head ldh = pad8(dim) + pad8(rot) elements, the part to rotate at pad8(dim).
 * Rotations.  Pairs (2i, 2i + 1) of the first rope_dims elements when interleaved, else (i, i + rope_dims / 2); rope is
 * [positions][rope_dims], per position rope_dims / 2 cosines, then as many sines. */

/* Elements of a cache row. */
int tilert_gqa_latent_row_len(int rank, int rot);
/* CTAs of latent_attn_op per part of the key range. */
int tilert_gqa_latent_blocks(int heads, int tokens, int rank, int rot, int f32);
/* Whether expanded_attn_op takes these sizes. */
int tilert_gqa_expanded_fits(int dim, int rot, int vdim);
/* From z [rows, ldz] f32 (query latent at 0, latent at off_c, key part at off_r): cq = rms(query latent) * q_gain, and
 * the cache rows of positions *pos + t. */
int tilert_gqa_latent_tokens_op(TgContext* ctx, const float* z, long long ldz, int q_rank, int off_c, int off_r,
                                const float* q_gain, const float* c_gain, float eps, int rows, int rank, int rot,
                                const float* rope, int positions, int rope_dims, int interleaved, const int* pos, int ring,
                                void* cq, long long ldq, void* cache, int f32, void* stream);
/* Projected queries [rows, ldq] f32, rotated.  lat NULL: out [rows, heads, pad16(dim) + pad16(rot)] (expanded form).  Else
 * (absorbed form) the unrotated part to out [heads, rows, pad8(dim)], the rotated part into lat [heads, rows, row] f32,
 * laid out like a cache row, whose first `rank` elements a product with the transposed key expansion fills. */
int tilert_gqa_latent_queries_op(TgContext* ctx, const float* q, long long ldq, int rows, int heads, int dim, int rot,
                                 const float* rope, int positions, int rope_dims, int interleaved, const int* pos, void* out,
                                 float* lat, int rank, int f32, void* stream);
/* Absorbed queries q [heads, tokens, row] f32 against the visible cache rows; token t is at *pos + t.  The key range is
 * shared by n_splits CTAs; part gets [heads, tokens, n_splits, rankp] unnormalised sums of latents, then [.., 2] (largest
 * score, sum of exponentials). */
int tilert_gqa_latent_attn_op(TgContext* ctx, const float* q, const void* cache, int tokens, int heads, int rank, int rot,
                              const int* pos, int window, int ring, float scale, int n_splits, float* part, int f32,
                              void* stream);
/* Parts -> out [heads, tokens, ldo]; sink [heads] or NULL: exp(sink) is one more term of the denominator. */
int tilert_gqa_latent_merge_op(TgContext* ctx, const float* part, int tokens, int heads, int n_splits, int rank, int rot,
                               const float* sink, void* out, long long ldo, int f32, void* stream);
/* out[t, h * vdim + v] = o[h, t, v] * sigmoid(gate[t, h]) (per_head) or sigmoid(gate[t, h * vdim + v]); gate NULL: 1. */
int tilert_gqa_gate_heads_op(TgContext* ctx, const float* o, int ldv, int rows, int heads, int vdim, const float* gate,
                             long long ldg, int per_head, void* out, long long ldo, int f32, void* stream);
/* The expanded form on bf16 tiles: kv [ring, heads * pad16(dim) | heads * pad16(vdim)] holds the keys and values of the
 * cache rows in use, the rotated key part is read from the cache.  Sink and gate as above, out [rows, heads * vdim]. */
int tilert_gqa_expanded_attn_op(TgContext* ctx, const void* q, const void* kv, const void* cache, int rows, int heads, int dim,
                                int rot, int vdim, int rank, const int* pos, int window, int ring, float scale,
                                const float* sink, const float* gate, long long ldg, int per_head, void* out, long long ldo,
                                void* stream);
/* One token: lat[h] = [w[h] q[h] | rotated part] with w [heads][rank][ldw] the transposed key expansion, and the cache
 * row of *pos from the latent c and the key part kr. */
int tilert_gqa_vec_absorb_op(TgContext* ctx, const float* q, int heads, int dim, int rank, int rot, const void* w, long long ldw,
                             const float* rope, int positions, int rope_dims, int interleaved, const float* c, const float* kr,
                             const float* c_gain, float eps, const int* pos, int ring, float* lat, void* cache, int f32,
                             void* stream);
/* One token: the merge of its parts, the value expansion w [heads][vdim][ldw] and the gate, out [heads * vdim]. */
int tilert_gqa_vec_value_op(TgContext* ctx, const float* part, int heads, int vdim, int rank, int rot, int n_splits,
                            const float* sink, const void* w, long long ldw, const float* gate, int per_head, float* out,
                            void* stream);

/* tilert_sample_op of tilert_b200.h (same kernel, same arguments). */
int tilert_gqa_sample_op(TgContext* ctx, const float* logits, long long logits_stride, int tokens, int vocab,
                         const float* config_dev, unsigned long long seed, unsigned long long* step_dev,
                         unsigned long long step_value, int* token_out, float* token_logprob_out, float* topn_logprob_out,
                         int* topn_index_out, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* TILERT_GQA_H_ */
