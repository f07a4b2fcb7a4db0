/*
 * cacheir_b200_hybrid.h -- C ABI of libcacheir_b200_hybrid.so: latent attention (Gutorax). Rows of a step as in
 * cacheir_b200_ragged.h.
 */
#ifndef CACHEIR_B200_HYBRID_H_
#define CACHEIR_B200_HYBRID_H_

#include "cacheir_b200_ragged.h"

#ifdef __cplusplus
extern "C" {
#endif

/* ---- latent attention: one cached row (latent | rotated key part) per token, shared by all heads ---------------- */
typedef struct {
  /* rows */
  const int32_t* positions;
  const int32_t* row_seg;
  const int32_t* cu_rows;
  const int32_t* page_table;
  int rows, segments, max_pages, page_size, num_slots;
  /* sizes */
  int heads, dim, rot_dim, vdim, kv_rank, window;
  float scale;
  /* cache: [num_slots, page_size, kv_rank + rot_dim] of `dtype` */
  void* pool;
  int dtype;
  int decode;               /* every segment has exactly one row (row i belongs to segment i) */
} cacheir_b200_latent_args;

/* down [rows, down_stride] = (latent before its norm | rotated part before its rotation), or NULL for a layer that reads
 * another layer's cache: the row goes to the pool. q [rows, q_stride] holds per head (dim | rot_dim): the rotated part
 * is turned and written to q_rot + row * q_rot_stride + head * q_rot_head_stride (in place when it points into q).
 * rope_table: float2 (cos, sin) [rope_positions, rot_dims / 2], rotate-half pairs (i, i + rot_dims/2). */
int cacheir_b200_latent_prepare(const cacheir_b200_latent_args* a, const void* down, long long down_stride, const float* norm_w,
                                float eps, const void* q, long long q_stride, void* q_rot, long long q_rot_stride,
                                int q_rot_head_stride, const float* rope_table, int rope_positions, int rot_dims, void* stream);
/* Any extents, float32 arithmetic: out [rows, heads*vdim] = gated attention output. uk [heads*dim, kv_rank],
 * uv [heads*vdim, kv_rank], sink [heads], gate [rows, gate_stride] before its sigmoid. */
int cacheir_b200_latent_attention_simple(const cacheir_b200_latent_args* a, const void* q, long long q_stride, const void* uk,
                                         const void* uv, const float* sink, const void* gate, long long gate_stride, void* out,
                                         void* stream);
/* Tensor-core form in latent space (bf16): q [rows, heads, kv_rank + rot_dim] (keys' up-projection already absorbed),
 * out [rows, heads, kv_rank]. `splits` (decode only, at most 8): CTAs that share a sequence's window; 0 = choose. */
int cacheir_b200_latent_attention_supported(int kv_rank, int rot_dim, int page_size, int dtype);
int cacheir_b200_latent_attention_splits(int rows, int heads, int window, int max_pages, int page_size);
int cacheir_b200_latent_attention(const cacheir_b200_latent_args* a, const void* q, const float* sink, void* out, int splits,
                                  void* stream);

/* First bounded wait of this library's kernels that gave up since the last reset (0: none). Synchronises. */
int cacheir_b200_hybrid_device_status(int reset);

#ifdef __cplusplus
}
#endif
#endif
