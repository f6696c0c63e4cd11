/* nqb200_mixers -- C ABI of the sequence-mixing kernels (sm_100a): input convolution fused with RMS norm, norms after
 * the residual sum, partial rotary embedding with a paged K/V store, chunk-masked attention with a score cap and a
 * sink or with sigmoid weights, retention, gated linear attention, minGRU, clamped GLU, per-layer token inputs, and
 * the skinny dense linears of decode steps with these steps inside.
 *
 * Conventions as in nqb200.h: plain device pointers, asynchronous on `stream`, status codes, nothing here
 * allocates.  `dtype` is the type of activations, weights and K/V caches: NQB200_BF16, or NQB200_F32 where
 * everything is computed and kept in 32 bits.  The residual stream, norm and convolution weights, gate biases
 * and recurrent states are always float.
 *
 * Tokens of a step are flattened; sequence b owns tokens cu[b] .. cu[b+1]-1, the first of which stands at
 * position pos0[b] of its sequence.  pos0[b] == 0 means that the sequence starts here: whatever its state slot
 * holds is taken as zero.  K/V of position p live in row (table[b * table_width + p / block_size] * block_size
 * + p % block_size) of the caches. */
#ifndef NQB200_MIXERS_H
#define NQB200_MIXERS_H

#include "nqb200.h"

#ifdef __cplusplus
extern "C" {
#endif

enum { NQB200_F32 = 2 };

typedef struct {
  const int32_t* cu;      /* [batch + 1] */
  const int32_t* pos0;    /* [batch] */
  const int32_t* slot;    /* [batch] row of the recurrent-state pools */
  const int32_t* table;   /* [batch, table_width] K/V blocks */
  int32_t batch, tokens, max_len, table_width, block_size;
} nqb200_batch;

/* x[t] = (accumulate ? x[t] : 0) + embed[ids[t]] + step.  ids or step may be NULL (that term is left out).
 * x float [tokens, width], embed [vocab, width] of `dtype`, step float [width]. */
int nqb200_stream_add(float* x, const int64_t* ids, const void* embed, const float* step, int accumulate,
                      int64_t tokens, int64_t width, int dtype, void* stream);

/* out[r] = RMSnorm(x[rows ? rows[r] : r]) * weight, rounded to dtype. */
int nqb200_rmsnorm_rows(const float* x, const int64_t* rows, const float* weight, void* out, int64_t n_rows,
                        int64_t width, float eps, int dtype, void* stream);

/* RMS norm in groups: the row is split into `groups` equal consecutive parts, each divided by its own root mean square,
 * and the whole multiplied by weight [width].
 * nqb200_group_norm_rows: out[r] = norm(x[rows ? rows[r] : r]), rounded to dtype.
 * nqb200_post_norm: x[t] = norm(alpha * x[t] + sum_{j < terms} y[t * terms + j]) in place; h[t] = x[t] rounded to dtype.
 * y [tokens * terms, width] is of y_dtype (NQB200_BF16 or NQB200_F32); terms = 0: nothing is added, y may be NULL. */
int nqb200_group_norm_rows(const float* x, const int64_t* rows, const float* weight, void* out, int64_t n_rows,
                           int64_t width, int64_t groups, float eps, int dtype, void* stream);
int nqb200_post_norm(float* x, const void* y, int y_dtype, int64_t terms, float alpha, const float* weight, void* h,
                     int64_t tokens, int64_t width, int64_t groups, float eps, int dtype, void* stream);

/* What a layer adds per token: out[t, i] = gelu_tanh(gate[t, i]) * table[ids[t] * table_stride + column + i], i < dim, and
 * x[t] += y[t] / rms(y[t]) * weight with h[t] = the sum rounded to dtype (y float [tokens, width]). */
int nqb200_gelu_table(const void* gate, const int64_t* ids, const void* table, int64_t table_stride, int64_t column,
                      void* out, int64_t tokens, int64_t dim, int dtype, void* stream);
int nqb200_add_normed(float* x, const float* y, const float* weight, void* h, int64_t tokens, int64_t width, float eps,
                      int dtype, void* stream);

/* h = RMSnorm(x) * weight; out[t, c] = h[t, c] + sum_j conv[j * width + c] h[t - taps + 1 + j, c], rounded to
 * dtype.  state float [slots, taps - 1, width] holds each sequence's last taps - 1 rows of h and is updated. */
int nqb200_rmsnorm_conv(const float* x, const float* weight, const float* conv, float* state, void* out,
                        const nqb200_batch* b, int64_t width, int64_t taps, float eps, int dtype, void* stream);

/* proj [tokens, stride] of dtype holds q (heads x dim at column q_off), k (kv_heads x dim at k_off) and v
 * (kv_heads x vdim at v_off).  q and k are rotated (pairs i, i + rot/2 of the first rot dimensions, angle
 * position * inv_freq[i]); q in place, k and v go to the caches [rows, kv_heads, dim | vdim]. */
int nqb200_rope_store(void* proj, void* k_cache, void* v_cache, const float* inv_freq, const nqb200_batch* b,
                      int64_t stride, int64_t q_off, int64_t k_off, int64_t v_off, int64_t heads, int64_t kv_heads,
                      int64_t dim, int64_t vdim, int64_t rot, int dtype, void* stream);

typedef struct {
  int32_t heads, kv_heads, dim, vdim;
  int32_t rot;             /* the first rot dimensions turn */
  int32_t interleaved;     /* pairs (2i, 2i + 1); else (i, i + rot/2) */
  const float* inv_freq;   /* [rot / 2] */
  const float* q_norm;     /* [dim] RMS norm over each head ahead of the rotation, or NULL */
  const float* k_norm;
  float eps;
} nqb200_rope;

/* nqb200_rope_store with both pair layouts and a norm ahead of the rotation.  v_off may be k_off: the values are then the
 * keys as projected.  k_cache NULL: k is turned in place and nothing is stored. */
int nqb200_norm_rope(void* proj, void* k_cache, void* v_cache, const nqb200_rope* r, const nqb200_batch* b, int64_t stride,
                     int64_t q_off, int64_t k_off, int64_t v_off, int dtype, void* stream);

typedef struct {
  int32_t heads, kv_heads, dim, vdim;
  int32_t chunk;          /* a query sees keys j <= i with j / chunk == i / chunk; <= 0: no chunks */
  float scale, softcap;   /* softcap <= 0: none */
  const float* sink;      /* [heads] or NULL */
  float out_scale;
  const float* temp;      /* [heads] factor of the scores, or NULL; sigmoid only */
  const float* bias;      /* [heads] added to the scores, or NULL; sigmoid only */
  int32_t sigmoid;        /* a key's weight is sigmoid(scale temp q.k + bias), not normalised: no softcap, no sink */
} nqb200_attention;

/* Attention of rotated q (rows of `q`, row stride q_stride, head h at column h * dim) over the paged caches of
 * cache_rows rows.  out[t * out_stride + h * vdim + c] = out_scale * o, rounded to dtype.  status (may be NULL): an int
 * on the device that takes NQB200_ERR_WAIT_TIMEOUT if a bounded wait gives up. */
int nqb200_chunk_attention(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, void* out,
                           int64_t out_stride, int64_t cache_rows, const nqb200_attention* a, const nqb200_batch* b, int* status, int dtype,
                           void* stream);

/* Retention.  proj holds q and k (heads x dim at q_off, k_off) and v (heads x vdim at v_off).
 * S <- decay[h] S + (dim^-1/2 k) v^T, o = S^T q, state float [slots, heads, dim, vdim].  o float [tokens, heads * vdim].
 * log_decay [tokens, heads * dim] (then decay is not read): gated linear attention, S <- diag(exp(log_decay)) S + ... */
int nqb200_retention(const void* proj, int64_t stride, int64_t q_off, int64_t k_off, int64_t v_off, const float* decay,
                     const float* log_decay, float* state, float* o, int64_t heads, int64_t dim, int64_t vdim, const nqb200_batch* b, int dtype,
                     void* stream);

/* Retention, or gated linear attention where rank > 0: then decay is not read, and the decays of channel c are
 * sigmoid(a2[c] . low + a2_bias[c])^(1 / tau), low the rank columns behind the gate. */
typedef struct {
  int32_t heads, dim, vdim;
  float eps, out_scale;
  const float* decay;     /* [heads] */
  const float* norm;      /* [vdim] weight of the norm over a head's output, or NULL */
  const float* inv_freq;  /* [rot / 2]; q and k turn in pairs (i, i + rot/2) inside nqb200_mixer_decode; other calls take */
  int32_t rot;            /* them turned (nqb200_norm_rope) */
  int32_t rank;
  float tau;
  const void* a2;         /* [heads * dim, rank] of dtype */
  const float* a2_bias;   /* [heads * dim] */
} nqb200_retention_desc;

/* Prompts (bf16): retention in chunkwise form with norm and gate.  proj holds q | k | v | gate from column off; the
 * result goes to act from column act_col.  chunk_states: scratch, 2 * nqb200_retention_chunks(tokens, batch) * heads *
 * dim * vdim floats. */
int nqb200_retention_prefill(const void* proj, int64_t stride, int64_t off, void* act, int64_t act_stride, int64_t act_col,
                             const nqb200_retention_desc* r, float* state, float* chunk_states, const nqb200_batch* b, void* stream);
int nqb200_retention_prefill_supported(const nqb200_retention_desc* r, int64_t stride, int64_t off, int64_t act_stride, int64_t act_col);
int64_t nqb200_retention_chunks(int64_t tokens, int64_t batch);

/* log_decay[t, c] = log(sigmoid(a2[c] . low[t] + bias[c])) / tau for c < channels; low [tokens, rank] with row stride
 * low_stride and a2 [channels, rank] of dtype. */
int nqb200_gla_log_decay(const void* low, int64_t low_stride, const void* a2, const float* bias, float* log_decay,
                         int64_t tokens, int64_t channels, int64_t rank, float tau, int dtype, void* stream);

/* Prompts (bf16): gated linear attention (rank > 0) in chunkwise form with norm and gate.  proj holds q | k | v | gate | low
 * from column off; the result goes to act from column act_col.  scratch: nqb200_gla_scratch() floats. */
int nqb200_gla_prefill(const void* proj, int64_t stride, int64_t off, void* act, int64_t act_stride, int64_t act_col,
                       const nqb200_retention_desc* r, float* state, float* scratch, const nqb200_batch* b, void* stream);
int nqb200_gla_prefill_supported(const nqb200_retention_desc* r, int64_t stride, int64_t off, int64_t act_stride, int64_t act_col);
int64_t nqb200_gla_scratch(const nqb200_retention_desc* r, int64_t tokens, int64_t batch);

/* out[t * out_stride + h * vdim + c] = out_scale * o / rms(o over the head) * weight[c] * silu(gate[t * gate_stride + h *
 * vdim + c]); weight [vdim] or NULL. */
int nqb200_head_norm_gate(const float* o, const void* gate, int64_t gate_stride, const float* weight, void* out, int64_t out_stride,
                          int64_t tokens, int64_t heads, int64_t vdim, float eps, float out_scale, int dtype, void* stream);

/* minGRU over proj [tokens, stride]: z, x and gate pre-activations at columns z_off, x_off, g_off.
 * z = sigmoid(zp + z_bias), u = xp + x_bias, candidate = u >= 0 ? u + 1/2 : sigmoid(u),
 * S <- (1 - z) S + z candidate, out = S silu(g).  state float [slots, width].
 * scratch: nqb200_mingru_scratch() floats (may be NULL where no sequence brings more than 128 tokens). */
int nqb200_mingru(const void* proj, int64_t stride, int64_t z_off, int64_t x_off, int64_t g_off, const float* z_bias,
                  const float* x_bias, float* state, void* out, int64_t width, float* scratch, const nqb200_batch* b,
                  int dtype, void* stream);
int64_t nqb200_mingru_scratch(int64_t tokens, int64_t batch, int64_t width);

/* out[t, i] = g sigmoid(1.702 g) (u + 1), g = min(gate_up[t, i], limit), u = clamp(gate_up[t, ff + i], -limit, limit). */
int nqb200_clamped_glu(const void* gate_up, void* out, int64_t tokens, int64_t ff, float limit, int dtype, void* stream);

/* ---- decode steps: at most 16 tokens, bf16 ---------------------------------------------------------------- */

enum { NQB200_DENSE_BF16 = 0, NQB200_DENSE_F32 = 1, NQB200_DENSE_RESIDUAL = 2 };

/* y = x w^T, x bf16 [M, K], w bf16 [N, K], M <= 16, K % 8 == 0.  mode: y as bf16, y as float, or float out = beta out + y. */
int nqb200_dense_decode(const void* x, const void* w, void* out, int64_t M, int64_t N, int64_t K, int mode, float beta, void* stream);

/* nqb200_gelu_table of the product (not rounded between): w [dim, K], out bf16 [M, dim]. */
int nqb200_dense_decode_gelu_table(const void* x, const void* w, const int64_t* ids, const void* table, int64_t table_stride,
                                   int64_t column, void* out, int64_t M, int64_t dim, int64_t K, void* stream);

/* w [2 ff, K] = gate rows, then up rows; out bf16 [M, ff] as nqb200_clamped_glu of the product (not rounded between). */
int nqb200_dense_decode_glu(const void* x, const void* w, void* out, int64_t M, int64_t ff, int64_t K, float limit, void* stream);

/* w [3 width, K] = z, x and gate rows; one token per sequence: product and nqb200_mingru update in one launch. */
int nqb200_dense_decode_mingru(const void* x, const void* w, const float* z_bias, const float* x_bias, float* state, void* out,
                               int64_t width, int64_t K, const nqb200_batch* b, void* stream);

/* One token per sequence: norm and rotation of the heads, K/V store and attention (columns q | k of proj from a_off, v from
 * v_off, output from column a_col of act), and retention or gated linear attention with norm and gate (columns q | k | v | g
 * [| low] from r_off, output from r_col), in one launch.  a or r may be NULL.  Sizes as nqb200_mixer_decode_supported says. */
int nqb200_mixer_decode(const void* proj, int64_t stride, void* act, int64_t act_stride, const nqb200_attention* a,
                        const nqb200_rope* rope, int64_t a_off, int64_t v_off, int64_t a_col, void* k_cache, void* v_cache,
                        const nqb200_retention_desc* r, int64_t r_off, int64_t r_col, float* state, const nqb200_batch* b, void* stream);
int nqb200_mixer_decode_supported(const nqb200_attention* a, const nqb200_retention_desc* r);

#ifdef __cplusplus
}
#endif
#endif
