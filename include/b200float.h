/*
 * b200float — C ABI of the B200 (sm_100a) kernels for models in floating point: linears, norms with a 32-bit residual
 * stream, depth averages, gated recurrences over vectors and matrices, attention over a paged latent cache or paged keys
 * and values, and the ends of a model.
 *
 * Conventions of b200int.h (status codes, borrowed pointers, nothing allocated or synchronised).  `dtype` is the type of
 * weights and of activations between kernels: B200F_BF16 (16-bit operands, 32-bit accumulation) or B200F_F32 (32-bit
 * throughout, no reduced-precision matrix mode).  Residual streams, norms, recurrent state, attention scores and
 * softmax are 32-bit for both.
 *
 * A linear whose K was split leaves `splits` partial sums [splits][rows][n] (fp32, `split_stride` elements apart); the
 * entry points that consume a linear's output take such a stack and add it in order, so results do not depend on timing.
 *
 * A batch is described as in the paged attention of b200int.h: 16-token pages, page_table [batch, pitch] of page ids,
 * kv_lens [batch] keys per sequence including the new tokens.  `seq_start` int32 [batch + 1] delimits every sequence's
 * new tokens; NULL means one new token per sequence (decode).  `slots` [batch] are rows of the per-sequence state.
 */
#ifndef B200FLOAT_H_
#define B200FLOAT_H_

#include "b200int.h"

#ifdef __cplusplus
extern "C" {
#endif

enum { B200F_F32 = 0, B200F_BF16 = 1 };
enum { B200F_ACT_NONE = 0, B200F_ACT_XIELU = 1, B200F_ACT_GATED_SILU = 2 };

/* ---- Linear: out[b][t, j] = act(sum_k x[b][t, k] * w[b][j, k]), b < batch.  Row pitches and batch strides in elements;
 * for B200F_BF16 every pitch and batch stride of x and w is a multiple of 8 and the bases are 16-byte aligned.
 * out_f32 selects a 32-bit output (always for B200F_F32).  splits > 1 (from b200f_gemm_splits; 32-bit output, no
 * activation): part s of K goes to out + s * split_stride.  act XIELU uses a = softplus(p), b = 1/2 + softplus(q):
 * a z^2 + z / 2 for z > 0, b (exp(z) - 1 - z) + z / 2 otherwise.  act GATED_SILU (bf16 output, n a multiple of 32): weight
 * rows alternate, 16 gates and 16 values, and out [m, n / 2] = silu(gate) * value. */
B200_API int b200f_gemm_splits(int64_t m, int64_t n, int64_t k, int64_t batch, int dtype);
B200_API int b200f_gemm(const void* x, const void* w, void* out, int dtype, int out_f32, int64_t m, int64_t n, int64_t k,
                        int64_t batch, int64_t x_pitch, int64_t x_bstride, int64_t w_pitch, int64_t w_bstride,
                        int64_t out_pitch, int64_t out_bstride, int splits, int64_t split_stride, int act, float act_a,
                        float act_b, b200_stream_t s);
B200_API int b200f_gemm_status(int* out_host, int reset);    /* synchronises with the device */

/* ---- Embedding row plus an optional bigram row (prev * mul_prev + cur * mul_cur) mod buckets; row `buckets` for
 * position 0.  prev_tokens int32 [slots]: the last token each sequence was given, read for the first new token and
 * replaced by the last one.  seq_ids int32 [tokens] (NULL for decode).  Writes fp32 [tokens, width] and, for bf16, the
 * rounded copy (pitch out_t_pitch). */
B200_API int b200f_embed_bigram(const void* table, const void* bigram, const int32_t* ids, const int32_t* positions,
                                const int32_t* seq_ids, const int32_t* seq_start, const int32_t* slots,
                                int32_t* prev_tokens, float* out, void* out_t, int dtype, int64_t tokens, int width,
                                int64_t vocab, int64_t buckets, int64_t mul_prev, int64_t mul_cur, int64_t out_t_pitch,
                                b200_stream_t s);

/* ---- End of a sublayer: r = x_in + rmsnorm(sum of y parts) * norm_w (+ add, one vector for all rows), all fp32
 * [rows, width]; x_in NULL is zero.  y2 (nullable): the normed quantity is the mean of rmsnorm(y) * w1 and
 * rmsnorm(sum of y2 parts) * w2 instead of y.
 * coef == NULL: x_out = r.  Otherwise a depth average over planes hist[0 .. planes-1] (plane_stride elements apart) and
 * r: r is stored to hist_out (nullable), x_out = sum coef[j] hist[j] + coef[planes] r.  final_w (nullable): x_out_t
 * receives rmsnorm(x_out) * final_w instead of x_out's copy (also for B200F_F32).  y == NULL: r = x_in (+ add). */
B200_API int b200f_sublayer_end(const float* y, int splits, int64_t split_stride, const float* y2, int splits2,
                                int64_t split_stride2, const float* w1, const float* w2, const float* x_in,
                                const float* norm_w, const float* add, float* x_out, void* x_out_t, const float* hist,
                                int planes, int64_t plane_stride, const float* coef, float* hist_out, const float* final_w,
                                int dtype, int64_t rows, int width, int64_t t_pitch, float eps, b200_stream_t s);

/* ---- xIELU on a stack of partial sums [rows, n] (see b200f_gemm for a and b). */
B200_API int b200f_xielu(const float* y, int splits, int64_t split_stride, void* out, int dtype, int64_t rows, int n,
                         int64_t out_pitch, float act_a, float act_b, b200_stream_t s);

/* ---- silu(gate) * value on a stack of partial sums [rows, y_pitch] whose columns alternate, 16 gates and 16 values;
 * n outputs per row. */
B200_API int b200f_gated_silu(const float* y, int splits, int64_t split_stride, int64_t y_pitch, void* out, int dtype,
                              int64_t rows, int n, int64_t out_pitch, b200_stream_t s);

/* ---- Gated recurrence (minGRU).  zug: parts of [tokens, 3 * width] pre-activations z | u | g; z += bias_z, u += bias_u;
 * S_t = (1 - sigmoid(z)) S_(t-1) + sigmoid(z) * cand(u), cand = u + 1/2 (u >= 0) or sigmoid(u); out = S_t * silu(g).
 * state fp32 [slots, width], taken as zero where the first new token has position 0. */
B200_API int b200f_mingru(const float* zug, int splits, int64_t split_stride, const float* bias_z, const float* bias_u,
                          float* state, const int32_t* slots, const int32_t* positions, const int32_t* seq_start,
                          void* out, int dtype, int64_t tokens, int batch, int width, int64_t out_pitch, b200_stream_t s);

/* ---- Between the projections of latent attention and its scores.  qd: parts of [tokens, heads * head_pitch (+ kv_rank +
 * rot_dim)]: per head dim unrotated and rot_dim rotated query entries, then, when the layer owns a cache
 * (dkv_norm != NULL), the latent and the shared key part.  Writes the unrotated queries [tokens, heads, qn_pitch], the
 * rotated ones into entries kv_rank .. of q_lat [tokens, heads, lat_pitch] (padding zeroed), and the normed latent and
 * the rotated key part into row out_loc of cache [.., lat_pitch].  rope fp32 [max_pos, rot_dims]: cos | sin. */
B200_API int b200f_latent_prepare(const float* qd, int splits, int64_t split_stride, int64_t qd_pitch,
                                  const int32_t* positions, const int32_t* out_loc, const float* rope, int rot_dims,
                                  int max_pos, const float* dkv_norm, float eps, void* qn, void* q_lat, void* cache,
                                  int dtype, int64_t tokens, int heads, int dim, int rot_dim, int kv_rank, int head_pitch,
                                  int qn_pitch, int lat_pitch, int64_t cache_rows, b200_stream_t s);

/* ---- Attention in the latent space: score(i, h, j) = scale * (q_lat[i, h] . cache[j]) over kv_rank + rot_dim entries,
 * visible keys i - window < j <= i (window 0: all j <= i), softmax whose denominator also has exp(sink[h]);
 * out[i, h] = sum_j p cache[j][0 .. kv_rank).  out [tokens, heads, out_pitch].
 * key_splits > 1 needs ws of b200f_latent_attn_ws_floats floats.  simple != 0 selects the plain kernel (always for
 * B200F_F32 and for sizes the tensor-core kernel does not take). */
B200_API size_t b200f_latent_attn_ws_floats(int64_t tokens, int heads, int kv_rank, int key_splits);
B200_API int b200f_latent_attn_splits(int64_t tokens, int batch, int max_q, int max_kv, int heads, int kv_rank,
                                      int rot_dim, int window, int dtype);
B200_API int b200f_latent_attn(const void* q_lat, const void* cache, const int32_t* page_table, int64_t table_pitch,
                               const int32_t* kv_lens, const int32_t* seq_start, const float* sink, void* out, int dtype,
                               int64_t tokens, int batch, int max_q, int heads, int kv_rank, int rot_dim, int lat_pitch,
                               int out_pitch, int window, float scale, int key_splits, float* ws, int simple,
                               b200_stream_t s);

B200_API int b200f_latent_attn_status(int* out_host, int reset);   /* as b200f_gemm_status: 5 copying warp, 6 consumer */

/* ---- Recurrences over a matrix per head, S_t = a_t S_(t-1) + k_t w_t^T, read-out S_t^T q_t, all in 32-bit.
 *   EXP    a = exp(f + m_(t-1) - m_t), w = exp(i - m_t) v, m_t = max(f + m_(t-1), i), m_0 = 0; n_t = a n_(t-1) + exp(i - m_t) k;
 *          den = max(|n_t . q|, exp(-m_t)) + 1e-6 (the read-out is not divided yet)
 *   SSD    a = exp(-exp(A_log) dt), w = dt v, dt = softplus(pre + dt_bias); skip[h] v is added to the read-out
 *   DELTA  q, k divided by sqrt(sum of squares + 1e-6); a = exp(-exp(A_log) softplus(pre + dt_bias)); w = beta (v - a S^T k)
 *
 * b200f_memory_prepare: `y` holds parts of the projections [tokens, y_pitch].  From column col0 on lie three segments
 * (segments[2 i] columns in heads of segments[2 i + 1]); they pass a causal convolution over `taps` tokens per channel
 * (conv_w [channels, taps], last column the current token's; conv_b nullable) and silu -- or nothing for taps 0 -- and
 * are written to `out` in dtype, each head padded to a multiple of 8 values (padding is not written).  conv_state fp32
 * [slots][taps - 1][channels]: the last inputs of each sequence, read and replaced.
 * Gates: columns gate_col_a / gate_col_b (+ head).  EXP: f and i, each cap * tanh((pre + bias) / cap) with biases gate_a /
 * gate_b, f then logsigmoid; norm_state fp32 [slots][heads][norm_dim + 1] holds n and, last, m, which is moved on here.
 * SSD and DELTA: dt from column a, gate_a = A_log, gate_b = dt_bias; DELTA: beta = sigmoid(column b).
 * gates fp32 [tokens][heads][4]: log a, write strength, exp(-m).
 *
 * b200f_memory_scan: rows as written above (q_off, k_off, v_off: columns of the first heads; head h of `heads` uses q / k
 * head h / (heads / qk_heads)); q_scale multiplies q.  state fp32 [slots][heads][dim][round8(vdim)], taken as zero where the
 * first new token has position 0.  out fp32 [tokens][heads * vdim], den fp32 [tokens][heads] (EXP).  dim <= 512.  max_q: most
 * new tokens of a sequence.  Prompts in bf16 run in chunks on the tensor cores (simple != 0: token by token); ws of
 * b200f_memory_scan_ws_bytes bytes.  The other two entries of a token's gates may be overwritten.
 *
 * b200f_memory_output: u = o / den (den nullable); groups of `group` values of a row are divided by their root mean square
 * (eps inside) and multiplied by norm_w (a gain per column, or norm_len == group gains for every group; with den, a group is
 * a head); the gate is the projection in column gate_col of y: silu(gate)
 * in front of the norm, or sigmoid(gate) or silu(gate) behind it. */
enum { B200F_MEMORY_EXP = 0, B200F_MEMORY_SSD = 1, B200F_MEMORY_DELTA = 2 };
enum { B200F_GATE_SILU_BEFORE = 0, B200F_GATE_SIGMOID_AFTER = 1, B200F_GATE_SILU_AFTER = 2 };
B200_API int b200f_memory_prepare(const float* y, int splits, int64_t split_stride, int64_t y_pitch, int64_t col0,
                                  const int32_t* segments, const float* conv_w, const float* conv_b, int taps,
                                  float* conv_state, const int32_t* slots, const int32_t* positions,
                                  const int32_t* seq_start, const int32_t* seq_ids, void* out, int64_t out_pitch, int dtype,
                                  int kind, int heads, int64_t gate_col_a, int64_t gate_col_b, const float* gate_a,
                                  const float* gate_b, float cap, float* gates, float* norm_state, int norm_dim,
                                  int64_t tokens, int batch, b200_stream_t s);
B200_API size_t b200f_memory_scan_ws_bytes(int64_t tokens, int batch, int max_q, int heads, int dim, int vdim, int kind, int dtype);
B200_API int b200f_memory_scan(const void* rows, int dtype, int64_t row_pitch, int64_t q_off, int64_t k_off, int64_t v_off,
                               int qk_heads, int heads, int dim, int vdim, int kind, float* gates, float q_scale,
                               const float* skip, float* state, float* norm_state, const int32_t* slots,
                               const int32_t* positions, const int32_t* seq_start, float* out, float* den, int64_t tokens,
                               int batch, int max_q, void* ws, int simple, b200_stream_t s);
B200_API int b200f_memory_scan_status(int* out_host, int reset);   /* as b200f_gemm_status: 7 a chunk's copies */
B200_API int b200f_memory_output(const float* o, const float* den, int heads, int vdim, int group, const float* y, int splits,
                                 int64_t split_stride, int64_t y_pitch, int64_t gate_col, int gate, const float* norm_w,
                                 int norm_len, float eps, void* out, int64_t out_pitch, int dtype, int64_t tokens,
                                 b200_stream_t s);

/* ---- Attention of grouped query heads: query head h reads key head h / (heads / kv_heads).
 * b200f_grouped_prepare: q, k, v from columns q_col, k_col, v_col of the projections; q and k divided by the root mean square
 * over all their heads and multiplied by q_norm / k_norm (nullable); q [tokens, heads, dim_pitch] and rows out_loc of the
 * caches [.., kv_heads, dim_pitch] and [.., kv_heads, vdim_pitch], padding zeroed.
 * b200f_grouped_attn: score scale * (q . k), visible keys i - window < j <= i (window 0: all j <= i), softmax;
 * out [tokens, out_pitch] has the heads side by side.  key_splits, ws and simple as for b200f_latent_attn. */
B200_API int b200f_grouped_prepare(const float* y, int splits, int64_t split_stride, int64_t y_pitch, int64_t q_col,
                                   int64_t k_col, int64_t v_col, const float* q_norm, const float* k_norm, float eps,
                                   const int32_t* out_loc, void* q, void* k_cache, void* v_cache, int dtype, int64_t tokens,
                                   int heads, int kv_heads, int dim, int vdim, int dim_pitch, int vdim_pitch,
                                   int64_t cache_rows, b200_stream_t s);
B200_API size_t b200f_grouped_attn_ws_floats(int64_t tokens, int heads, int vdim, int key_splits);
B200_API int b200f_grouped_attn_splits(int64_t tokens, int batch, int max_q, int max_kv, int heads, int kv_heads, int dim,
                                       int vdim, int window, int dtype);
B200_API int b200f_grouped_attn(const void* q, const void* k_cache, const void* v_cache, const int32_t* page_table,
                                int64_t table_pitch, const int32_t* kv_lens, const int32_t* seq_start, void* out, int dtype,
                                int64_t tokens, int batch, int max_q, int heads, int kv_heads, int dim, int vdim,
                                int dim_pitch, int vdim_pitch, int64_t out_pitch, int window, float scale, int key_splits,
                                float* ws, int simple, b200_stream_t s);

/* ---- Row-wise arg-max of fp32 logits, the lowest index wins ties. */
B200_API int b200f_argmax(const float* logits, int64_t rows, int64_t n, int64_t pitch, int32_t* out_idx, b200_stream_t s);

#ifdef __cplusplus
}
#endif
#endif /* B200FLOAT_H_ */
