/*
 * cacheir_b200_experts.h -- C ABI of libcacheir_b200_experts.so: attention over cached rows that hold key and value, and
 * mixtures of experts (Topunex, Rekodra). Rows of a step as in cacheir_b200_ragged.h.
 */
#ifndef CACHEIR_B200_EXPERTS_H_
#define CACHEIR_B200_EXPERTS_H_

#include "cacheir_b200_ragged.h"

#ifdef __cplusplus
extern "C" {
#endif

/* ---- tied attention: grouped-query attention whose cached row is key and value at once ------------------------------
 * A row of `width` columns per key/value head: its first `dim` columns are the value, columns key_from .. width - 1 the key
 * (the two may overlap), and inv_rms beside it a factor of every product with the row:
 *   q . key = (q . row[key_from:]) * inv_rms
 * so that a key's normalisation costs no second copy. cacheir_b200_tied_prepare makes two kinds of rows of a key with
 * `rot_dims` rotated entries:
 *   values are the keys:  (k as projected | its first rot_dims entries rotated),  key_from = rot_dims
 *   values of their own:  (v | first rot_dims entries of k rotated | the rest as projected),  key_from = dim
 * score = cap * tanh(q . key * scale / cap) (cap <= 0: no cap). A row at position i sees j <= i with i - j < window or
 * j < keep_first. exp(sink[head]) joins the denominator (sink NULL: nothing does). */
typedef struct {
  /* rows */
  const int32_t* positions;
  const int32_t* row_seg;
  const int32_t* cu_rows;
  const int32_t* page_table;
  int rows, segments, max_pages, page_size, num_slots;
  /* sizes */
  int heads, kv_heads, dim, width, key_from, window, keep_first;
  float scale, cap;
  float reach;              /* |q . key| never exceeds it, before the scale; 0: no such bound is known */
  /* cache: rows [num_slots, kv_heads, page_size, width] of `dtype`, inv_rms [num_slots, kv_heads, page_size] */
  void* pool;
  float* inv_rms;
  const float* sink;
  int dtype;
  int decode;               /* every segment has exactly one row (row i belongs to segment i) */
} cacheir_b200_tied_args;

/* q [rows, q_stride] heads*d columns, k [rows, k_stride] kv_heads*d columns, v [rows, v_stride] kv_heads*dim columns, as
 * projected (v NULL: the values are the keys, d = dim; else d = width - dim). Queries and keys are divided by their root mean
 * square, per head or (`whole`) over all heads at once, multiplied by q_weight and k_weight (NULL: ones; d entries, or one for
 * every column with `whole`), and rotated (rotate-half pairs on the first rot_dims entries of a head). The cache rows go to the
 * pool; queries to q_out [rows, heads, width - lead] as what a cached row is multiplied with (key weights of unrotated
 * entries included): key_from zeros, then the key's columns, without the first lead = key_from / 64 * 64 zeros.
 * rope_table: float2 (cos, sin) [rope_positions, rot_dims / 2]. */
int cacheir_b200_tied_prepare(const cacheir_b200_tied_args* a, const void* q, long long q_stride, const void* k, long long k_stride,
                              const void* v, long long v_stride, int rot_dims, int whole, const float* q_weight, const float* k_weight,
                              float eps, const float* rope_table, int rope_positions, void* q_out, void* stream);
/* out [rows, heads*dim] = attention * sigmoid(gate), gate [rows, gate_stride] before its sigmoid (NULL: no gate).
 * simple: any extents, float32 arithmetic. prompt: tiles of neighbouring tokens on the tensor cores. step: one row per
 * segment, `splits` CTAs (at most 8, 0 = choose) share a sequence. */
int cacheir_b200_tied_attention_simple(const cacheir_b200_tied_args* a, const void* q, const void* gate, long long gate_stride, void* out,
                                       void* stream);
int cacheir_b200_tied_prompt_supported(int heads, int kv_heads, int dim, int width, int key_from, int page_size, int dtype);
int cacheir_b200_tied_attention_prompt(const cacheir_b200_tied_args* a, const void* q, const void* gate, long long gate_stride, void* out,
                                       void* stream);
int cacheir_b200_tied_step_supported(int heads, int kv_heads, int dim, int width, int key_from, int page_size, int dtype);
int cacheir_b200_tied_step_splits(int rows, int heads, int kv_heads, int window, int keep_first, int max_pages, int page_size);
int cacheir_b200_tied_attention_step(const cacheir_b200_tied_args* a, const void* q, const void* gate, long long gate_stride, void* out,
                                     int splits, void* stream);

/* ---- mixtures of experts ----------------------------------------------------------------------------------------------
 * route: per row of logits [rows, stride] the `top` experts with the largest values (lower index first among equals),
 * weight = sigmoid(logit) * scale. A softmax rule chooses by softmax + correction instead, within the `keep` groups of
 * neighbours whose largest choice score is largest, and weighs with softmax * scale. Logits experts .. experts + identity - 1
 * stand for the token itself (PLACE_SELF instead of a place). The rows x top choices get places 0.. in expert order:
 *   cu [experts + 1] first place of every expert; token_of [rows*top] row of a place; place_of, weight, chosen [rows, top]
 * Rows with row_seg < 0 choose nothing (place_of = -1). `counters`: experts + 1 zeroed ints, left zeroed. With `placed`
 * [rows*top, row_bytes] every row of x [rows, row_bytes] is also copied to its places (multiples of 16 bytes). */
#define CACHEIR_B200_PLACE_NONE (-1)
#define CACHEIR_B200_PLACE_SELF (-2)
typedef struct {
  int softmax;              /* 0: sigmoid of the logit, no correction and no groups */
  int identity;
  int groups, keep;
  const float* correction;  /* [experts + identity] or NULL */
  float scale;
} cacheir_b200_route_rule;
int cacheir_b200_route(const float* logits, long long stride, const int32_t* row_seg, int rows, int experts, int top,
                       const cacheir_b200_route_rule* rule, int32_t* counters, int32_t* cu, int32_t* token_of, int32_t* place_of, float* weight, int32_t* chosen,
                       const void* x, void* placed, int row_bytes, void* stream);
/* Y[place] = f(X[.] W_e^T) for the places of every expert e, whose W rows start at e*w_batch_rows. X rows are places; with
 * place_of [x_rows, top] they are the step's rows (at most cacheir_b200_grouped_all_rows() of them). a->T places at most,
 * a->batch experts. Epilogues: BF16, SWIGLU, CLAMPED_GLU. Strides must be multiples of 8 elements. */
int cacheir_b200_grouped_all_rows(void);
int cacheir_b200_grouped_gemm(const cacheir_b200_dense_args* a, const int32_t* cu, const int32_t* place_of, int top, int x_rows, void* stream);
/* The same product without its epilogue in float32 arithmetic, any extents; X rows are places, or token_of[place]. */
int cacheir_b200_grouped_simple(const void* x, const void* w, void* y, const int32_t* cu, const int32_t* token_of, int places, int experts,
                                int N, int K, long long w_stride, long long x_stride, long long y_stride, int dtype, void* stream);
/* m = sum_k weight[t, k] * y[place_of[t, k]] + shared[t] (shared may be NULL); residual += m / sqrt(mean(m^2) + eps) * w,
 * then next_mode (NONE or COPY) */
int cacheir_b200_combine_residual_rms(float* residual, const void* y, const int32_t* place_of, const float* weight, int top,
                                      const void* shared, const float* w, float eps, int rows, int width, int next_mode, void* next_out,
                                      int dtype, void* stream);

/* residual += sum over a row's choices of weight * (y[place], or self[t] for PLACE_SELF) + shared[t] * sigmoid(shared_gate[t *
 * shared_gate_stride]) (shared NULL: none; shared_gate NULL: factor one), then next_mode (NONE, COPY or RMS) */
int cacheir_b200_combine_residual(float* residual, const void* y, const int32_t* place_of, const float* weight, int top, const void* self,
                                  const void* shared, const float* shared_gate, long long shared_gate_stride, int rows, int width, int next_mode,
                                  const float* next_w, const float* next_b, float next_alpha, void* next_out, int dtype, void* stream);

/* First bounded wait of this library's kernels that gave up since the last reset (0: none). Synchronises. */
int cacheir_b200_experts_device_status(int reset);

#ifdef __cplusplus
}
#endif
#endif
