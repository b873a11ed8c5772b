/*
 * l3ci_mixers.h — C ABI of libl3ci_mixers.so: the layer parts of decoders other than Llama-3 (latent, differential and
 * windowed attention, linear recurrences, mixture of experts, norms over a 32-bit residual stream, activations).
 *
 * Conventions of l3ci_b200.h: device pointers, strides in ELEMENTS, asynchronous on `stream`, returns an
 * l3ci_status; detail text in l3ci_mixers_last_error().  `dtype` is the storage type of activations and caches:
 * L3CI_BF16 or L3CI_F32 (tensors the comments call fp32 are fp32 in both).  Arithmetic is fp32 in both.
 */
#ifndef L3CI_MIXERS_H_
#define L3CI_MIXERS_H_

#include "l3ci_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

typedef enum l3ci_dtype { L3CI_BF16 = 0, L3CI_F32 = 1 } l3ci_dtype;

L3CI_API const char* l3ci_mixers_last_error(void);
L3CI_API int l3ci_mixers_set_programmatic_launch(int on);

/* Residual add fused into a dynamic-tanh norm (no statistics):  x += y;  out = tanh(alpha * x) * weight + bias.
 * x is the fp32 residual stream [rows, width], updated in place; y (dtype) may be null; with `tokens` (int64
 * [rows]) the residual starts as x = table[tokens] (dtype [vocab, width]) instead, y null.  weight, bias: fp32. */
L3CI_API int l3ci_add_dyn_tanh(const void* y, const int64_t* tokens, const void* table, int64_t vocab, float* x,
                               const float* weight, const float* bias, float alpha, void* out, int64_t rows,
                               int64_t width, int32_t dtype, l3ci_stream_t stream);

/* One pass over the rows of the fp32 residual stream x [rows, width] between two sublayers:
 *   y = sum over p < parts of part_weights[row, p] * y[part_rows[row, p], :]
 *       (part_weights null: 1; part_rows null: row * parts + p; y null: nothing is added)
 *   x = (reset ? 0 : x) + (post_w ? layer_norm(y) * post_w + post_b : y) + step
 *   out[row * out_stride + ...] = pre_w ? layer_norm(x) * pre_w + pre_b : x        (out null: not written)
 * With `tokens` (int64 [rows]) the stream starts instead as x = table[tokens] * embed_scale + s, where s is the sinusoidal
 * vector of the row's position positions[row / T] + row % T: entries 2i, 2i + 1 are sin, cos of position * freqs[i]
 * (freqs null: no s); x0 (null: not wanted) receives a copy of it in the storage type.
 * Weights, biases, step, part_weights: fp32.  y is of y_dtype, table / out / x0 of dtype.  layer_norm divides the
 * deviation from the mean by sqrt(mean of its square + eps). */
typedef struct l3ci_residual_norm_args {
  float* x;
  const void* y;
  const float* part_weights;
  const int32_t* part_rows;
  const float *post_w, *post_b, *step, *pre_w, *pre_b;
  void* out;
  const int64_t* tokens;
  const void* table;
  const double* freqs;
  const int32_t* positions;
  void* x0;
  int64_t out_stride, x0_stride, vocab, rows, width;
  int32_t parts, reset, T, dtype, y_dtype;
  float eps, embed_scale;
  l3ci_stream_t stream;
} l3ci_residual_norm_args;

L3CI_API int l3ci_residual_norm(const l3ci_residual_norm_args* args);

/* out = z * Phi(z) (exact gelu, erf form), n elements, in place allowed. */
L3CI_API int l3ci_gelu(const void* z, void* out, int64_t n, int32_t dtype, l3ci_stream_t stream);
/* out = tanh(z), n elements, in place allowed. */
L3CI_API int l3ci_tanh(const void* z, void* out, int64_t n, int32_t dtype, l3ci_stream_t stream);

/* Gated feed-forward activation of rows gu = [gate (ff) | up (ff)], out [rows, ff]:
 *   limit == 0: silu(gate) * up;   limit > 0: with g = min(gate, limit), u = clamp(up, -limit, limit):
 *   g * sigmoid(alpha * g) * (u + 1). */
L3CI_API int l3ci_gated_act(const void* gu, void* out, int64_t rows, int64_t ff, float limit, float alpha, int32_t dtype,
                            l3ci_stream_t stream);

/* A row [q | k | v] of a fused projection (widths q_width, k_width, v_width, one behind the other): RMS norm over the
 * whole of q (in place) and over the whole of k, weights q_norm and k_norm (fp32), then k and v into the caches at
 * p = positions[b] + t, as l3ci_kv_cache_write does. */
L3CI_API int l3ci_qk_norm_cache(void* qkv, int64_t stride, int64_t q_width, int64_t k_width, int64_t v_width,
                                const float* q_norm, const float* k_norm, float eps, void* cache_k, int64_t k_sb,
                                int64_t k_st, void* cache_v, int64_t v_sb, int64_t v_st, int64_t cache_len,
                                const int32_t* positions, int32_t B, int32_t T, int32_t dtype, l3ci_stream_t stream);

/* Token shift: out[s, row, :] = h[row] + (h[row - 1] - h[row]) * mu[s, :] for s < n_mix; rows are (sequence, token),
 * h[row - 1] of a sequence's first token is `last` (dtype [.., width], one row per sequence, last_sb apart; taken as zeros at
 * positions[b] == 0), which then receives h of its last token.  mu: fp32 [n_mix, width]. */
L3CI_API int l3ci_token_shift(const void* h, const float* mu, void* last, int64_t last_sb, const int32_t* positions, void* out,
                              int32_t n_mix, int32_t B, int32_t T, int64_t width, int32_t dtype, l3ci_stream_t stream);

/* Inputs of the gated delta rule from rows p = [q (G*D) | k (G*D) | v (H*V)] (dtype, p_st apart), each channel through a
 * causal convolution over its last `taps` inputs (conv: fp32 [taps][2*G*D + H*V], the last row is the current token's) and
 * silu; q and k made unit vectors per head (x / sqrt(sum x^2 + unit_eps)), q times D^-0.5:
 *   qk_out fp32 [rows][2][G][D],  v_out dtype [rows][H][V],
 *   beta_out fp32 [rows][H] = sigmoid(b),   decay_out fp32 [rows][H][D] = exp(-exp(a_log[h]) * softplus(a + dt_bias)).
 * `tail` holds a sequence's last taps - 1 inputs (dtype [taps - 1][2*G*D + H*V], tail_sb apart), zeros at positions[b] == 0; it
 * is only read (l3ci_recurrent_scan moves it on). */
typedef struct l3ci_delta_inputs_args {
  const void *p, *b, *a;
  const float *conv, *a_log, *dt_bias;
  const void* tail;
  const int32_t* positions;
  float *qk_out, *beta_out, *decay_out;
  void* v_out;
  int64_t p_st, b_st, a_st, tail_sb;
  int32_t B, T, H, G, D, V, taps, dtype;
  float unit_eps;
  l3ci_stream_t stream;
} l3ci_delta_inputs_args;

L3CI_API int l3ci_delta_inputs(const l3ci_delta_inputs_args* args);

/* Linear recurrence over a matrix state S [D, V] per (sequence, head), fp32, then the head's output norm and gate:
 *   kind 0 (gated delta rule): S <- g * S (rows);  u = beta * (v - S^T k);  S <- S + k u^T;  o = S^T q
 *        q, k, g, beta fp32 (beta [rows, H]); state head h reads q / k head h / (H / G)
 *   kind 1 (time mixing):      o = (S + diag(bonus) k v^T)^T q;  S <- g * S + k v^T,  g = exp(-exp(g_raw + g_bias))
 *        q, k, g_raw of dtype; g_bias, bonus fp32 [H, D]; G == H
 *   out[row, h, :] = o / sqrt(mean(o^2) + eps) * norm[h * norm_sh + :] * act(gate[row, h, :]),
 *        act: 0 sigmoid, 1 silu.
 * The state starts at zero where positions[b] == 0, else from `state` (fp32 [H][D][V] per sequence, state_sb apart), which
 * receives the state after the last token.  tail != null: the convolution inputs of l3ci_delta_inputs (rows `conv_in`) are
 * moved on by T tokens. */
typedef struct l3ci_recurrent_scan_args {
  const void *q, *k, *v, *g;
  const float *beta, *bonus, *g_bias, *norm;
  const void* gate;
  float* state;
  void* out;
  const void* conv_in;
  void* tail;
  const int32_t* positions;
  int32_t* status;            /* optional device word: L3CI_ERR_DEVICE_WAIT when a bounded wait runs out          */
  int64_t qk_st, qk_sh, v_st, v_sh, g_st, g_sh, gate_st, gate_sh, out_st, out_sh, norm_sh, state_sb, conv_st, tail_sb;
  int32_t kind, B, T, H, G, D, V, act, taps, dtype;
  float eps;
  l3ci_stream_t stream;
} l3ci_recurrent_scan_args;

L3CI_API int l3ci_recurrent_scan(const l3ci_recurrent_scan_args* args);

/* Mixture of experts.  Route: of the fp32 logits [rows, E] + bias [E] the `top` largest of a token (ties: the smaller index),
 * weights = softmax over these; experts, ranks int32 [rows, top] (rank: place of the pair among the pairs of its expert),
 * weights fp32.  counts int32 [E] is set to the experts' pairs. */
L3CI_API int l3ci_moe_route(const float* logits, const float* bias, int32_t* experts, int32_t* ranks, float* weights,
                            int32_t* counts, int64_t rows, int32_t n_experts, int32_t top, l3ci_stream_t stream);
/* Rows sorted by expert: out[at] = h[row], at = (sum of counts of smaller experts) + rank; part_rows[row, j] = at. */
L3CI_API int l3ci_moe_gather(const void* h, const int32_t* experts, const int32_t* ranks, const int32_t* counts, void* out,
                             int32_t* part_rows, int64_t rows, int64_t width, int32_t n_experts, int32_t top, int32_t dtype,
                             l3ci_stream_t stream);
/* Products of the sorted rows x [rows, K] with their experts' matrices w.
 *   gated == 0: w [E, N, K], out [rows, N] = x w^T.
 *   gated == 1: w [E, 2, N, K] (gate, up), out [rows, N] = the clamped activation of l3ci_gated_act of x gate^T, x up^T.
 * variant 0: choose; 1: plain (any size, both types); 2: tcgen05.  status: as in l3ci_mixer_attn_args. */
typedef struct l3ci_moe_gemm_args {
  const void *x, *w;
  void* out;
  const int32_t* counts;
  int32_t* status;
  int64_t rows;
  int32_t K, N, n_experts, gated, dtype, variant;
  float limit, alpha;
  l3ci_stream_t stream;
} l3ci_moe_gemm_args;

L3CI_API int l3ci_moe_gemm(const l3ci_moe_gemm_args* args);
/* The variant the call would run (1 or 2), -1 for arguments it would refuse. */
L3CI_API int l3ci_moe_gemm_variant(const l3ci_moe_gemm_args* args);

/* One token row qd = [H heads of (dim, rot_dim) | rank | rot_dim] of the fused query / latent projection:
 *   the rot_dim part of every query head is rotated in place (rotate-half pairs i, i + rot_dim/2);
 *   cache[b, p] = [ rms_norm(latent) * norm_weight | rotated key part ]  at p = positions[b] + t.
 * Token t of sequence b is row b*T + t of qd.  `table` is fp32 [table_rows, rot_dim]: (cos, sin) of pair 0, pair 1,
 * ... per position.  A position outside the table or the cache is skipped. */
L3CI_API int l3ci_latent_cache(void* qd, int64_t qd_stride, const float* table, int64_t table_rows,
                               const float* norm_weight, float eps, void* cache, int64_t cache_sb, int64_t cache_st,
                               int64_t cache_len, const int32_t* positions, int32_t B, int32_t T, int32_t H, int32_t dim,
                               int32_t rot_dim, int32_t rank, int32_t dtype, l3ci_stream_t stream);

/* k and v columns of a fused projection row into the caches, unrotated: cache_k[b, p, :] = src[row, k_col : + k_width],
 * cache_v[b, p, :] = src[row, v_col : + v_width],  p = positions[b] + t. */
L3CI_API int l3ci_kv_cache_write(const void* src, int64_t src_stride, int64_t k_col, int64_t k_width, int64_t v_col,
                                 int64_t v_width, void* cache_k, int64_t k_sb, int64_t k_st, void* cache_v, int64_t v_sb,
                                 int64_t v_st, int64_t cache_len, const int32_t* positions, int32_t B, int32_t T,
                                 int32_t dtype, l3ci_stream_t stream);

/* Causal attention of T >= 1 new tokens per sequence over cached keys and values.
 *
 * Query head h of H reads key/value head h / (H / G).  A query (and key) is one vector in two parts of sizes Da and
 * Db (Db may be 0): score = (qa . ka + qb . kb) * scale * temperature(p), then, with softcap > 0,
 * softcap * tanh(score / softcap).  temperature(p) = 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)
 * (temp_every 0: 1), then, with bias_range > 0, minus the distance bias 2^(-bias_range (h + 1) / H) * (p - j).  Token t of
 * sequence b is at p = positions[b] + t and sees keys j <= p with p - j < window (window 0: all) or j < keep_first.  sink != 0:
 * the softmax has one more term in its denominator, a score of 0 without a value.  Window, bias and sink: one map only.
 *
 * maps == 1: out[b, t, h, 0:Dv] = softmax(scores) v.
 * maps == 2 (differential attention): a query head is [map 1, map 2] of Da each, a key head likewise, Db = 0; with
 * a1, a2 the maps' outputs over the same values, o = a1 - lambda * a2, out = o / sqrt(mean(o^2) + eps) * post *
 * sigmoid(gate[b, t, h]) (gate null: no gate). */
typedef struct l3ci_mixer_attn_args {
  const void *qa, *qb, *ka, *kb, *v;
  const void* gate;
  void* out;
  const int32_t* positions;   /* int32 [B] on the device                                                        */
  void* scratch;              /* l3ci_mixer_attention_scratch_bytes; may be null when that is 0                   */
  size_t scratch_bytes;
  int32_t* status;            /* optional device word: L3CI_ERR_DEVICE_WAIT when a bounded wait runs out          */
  int64_t qa_sb, qa_st, qa_sh, qb_sb, qb_st, qb_sh;
  int64_t ka_sb, ka_st, ka_sh, kb_sb, kb_st, kb_sh, v_sb, v_st, v_sh;
  int64_t o_sb, o_st, o_sh, g_sb, g_st;
  int32_t dtype, B, T, H, G, maps, Da, Db, Dv;
  int32_t n_keys;             /* rows of k and v that may be read (cache length, or start_pos + T)                */
  int32_t start_pos;          /* host-known positions[] of every sequence, or -1 (device only)                    */
  int32_t variant;            /* 0: choose; 1: a CTA per query (any size, both types); 2: mma.sync, keys split over
                                 CTAs; 3: tcgen05 (128 query rows per CTA)                                         */
  int32_t window, keep_first, sink;
  float scale, softcap, temp_coef, temp_every, lambda, post, eps, bias_range;
  l3ci_stream_t stream;
} l3ci_mixer_attn_args;

L3CI_API int l3ci_mixer_attention(const l3ci_mixer_attn_args* args);
/* Bytes of scratch the call wants (0: none).  Depends on the device's SM count. */
L3CI_API size_t l3ci_mixer_attention_scratch_bytes(const l3ci_mixer_attn_args* args);
/* The variant the call would run (1, 2 or 3), -1 for arguments it would refuse. */
L3CI_API int l3ci_mixer_attention_variant(const l3ci_mixer_attn_args* args);

#ifdef __cplusplus
}
#endif
#endif /* L3CI_MIXERS_H_ */
