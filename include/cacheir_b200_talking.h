/*
 * cacheir_b200_talking.h -- C ABI of libcacheir_b200_talking.so: attention whose heads mix their scores before the softmax
 * (Zimorax). Rows of a step as in cacheir_b200_ragged.h.
 */
#ifndef CACHEIR_B200_TALKING_H_
#define CACHEIR_B200_TALKING_H_

#include "cacheir_b200_ragged.h"

#ifdef __cplusplus
extern "C" {
#endif

/* score_h = sum_g talk[h, g] (q_g . key) scale, every head g against the key of its own key/value head; p = exp(score) / (1 +
 * sum exp(score)); a row at position i sees j <= i with i - j < window. A cached token has one row of keys and one of values, all
 * key/value heads side by side. */
typedef struct {
  /* rows */
  const int32_t* positions;
  const int32_t* row_seg;
  const int32_t* cu_rows;
  const int32_t* page_table;
  int rows, segments, max_pages, page_size, num_slots;
  /* sizes */
  int heads, kv_heads, dim, vdim, window;
  float scale;
  const float* talk;        /* [heads, heads] */
  /* cache: keys [num_slots, page_size, kv_heads*dim], values [num_slots, page_size, kv_heads*vdim] of `dtype` */
  void* keys;
  void* values;
  int dtype;
  int decode;               /* every segment has exactly one row (row i belongs to segment i) */
} cacheir_b200_talking_args;

/* q, k, v as projected. Queries and keys are rotated (rotate-half pairs on the first rot_dims entries of a head; rope_table: float2
 * (cos, sin) [rope_positions, rot_dims / 2]), values divided by their root mean square per head; keys and values go to the cache.
 * q_out [rows, heads, dim]: rotated queries. With `mixed`, [rows, heads, kv_heads*dim]: what head h multiplies a whole cached key
 * row with to get its mixed score, for every key/value head the sum of talk[h, g] q_g over its heads g, with the sign of the scale (dim % 8 == 0). */
int cacheir_b200_talking_prepare(const cacheir_b200_talking_args* a, const void* q, long long q_stride, const void* k, long long k_stride,
                                 const void* v, long long v_stride, int rot_dims, const float* rope_table, int rope_positions, float eps,
                                 int mixed, void* q_out, void* stream);
/* out [rows, heads*vdim]. simple: any extents, float32 arithmetic, rotated queries. step: one row per segment, rotated queries,
 * `splits` CTAs (at most 8, 0 = choose) share a sequence. prompt: tiles of neighbouring tokens, mixed queries. */
int cacheir_b200_talking_simple(const cacheir_b200_talking_args* a, const void* q, void* out, void* stream);
int cacheir_b200_talking_step_supported(int heads, int kv_heads, int dim, int vdim, int page_size, int dtype);
int cacheir_b200_talking_step_splits(int rows, int heads, int kv_heads, int dim, int vdim, int window, int max_pages, int page_size);
int cacheir_b200_talking_step(const cacheir_b200_talking_args* a, const void* q, void* out, int splits, void* stream);
int cacheir_b200_talking_prompt_supported(int heads, int kv_heads, int dim, int vdim, int page_size, int dtype);
int cacheir_b200_talking_prompt(const cacheir_b200_talking_args* a, const void* mixed_q, void* out, void* stream);

/* First bounded wait of this library's kernels that gave up since the last reset (0: none). Synchronises. */
int cacheir_b200_talking_device_status(int reset);

#ifdef __cplusplus
}
#endif
#endif
