/*
 * l3ci_mixers.h — C ABI of libl3ci_mixers.so: the layer parts of decoders other than Llama-3 (latent attention,
 * differential attention, a dynamic-tanh norm over a 32-bit residual stream, the exact gelu).
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

/* out = z * Phi(z) (exact gelu, erf form), n elements, in place allowed. */
L3CI_API int l3ci_gelu(const void* z, void* out, int64_t n, int32_t dtype, l3ci_stream_t stream);

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
 * (temp_every 0: 1).  Token t of sequence b is at p = positions[b] + t and sees keys j <= p.
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
  float scale, softcap, temp_coef, temp_every, lambda, post, eps;
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
