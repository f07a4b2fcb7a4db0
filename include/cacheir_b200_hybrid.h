/*
 * cacheir_b200_hybrid.h -- C ABI of libcacheir_b200_hybrid.so: the kernels of decoder families whose layers mix latent
 * attention with linear recurrences (Gutorax). Conventions are those of cacheir_b200.h: device pointers and sizes only,
 * no allocation, no synchronisation, 0 / positive cudaError_t / negative CACHEIR_B200_E* return values.
 *
 * A step runs `rows` token rows of `segments` sequences. Rows of one sequence are neighbours in position order:
 *   cu_rows   [segments + 1]  first row of every sequence (cu_rows[segments] = rows in use; later rows are padding)
 *   row_seg   [rows]          sequence of a row, -1 for padding
 *   positions [rows]          position of a row in its sequence
 *   page_table [segments, max_pages], slots [segments]: where the sequence's cache pages and recurrent state live
 * The residual stream is float32; activations are `dtype` (F32 or BF16); norm weights are float32.
 */
#ifndef CACHEIR_B200_HYBRID_H_
#define CACHEIR_B200_HYBRID_H_

#include "cacheir_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

/* What a kernel that finishes the residual stream leaves as the next operator's input */
#define CACHEIR_B200_NEXT_NONE 0
#define CACHEIR_B200_NEXT_COPY 1   /* the residual itself, rounded to the activation type */
#define CACHEIR_B200_NEXT_DYT 2    /* tanh(alpha * residual) * w + b                      */

/* Epilogues of cacheir_b200_dense_gemm */
#define CACHEIR_B200_DENSE_BF16 0        /* y                                                        */
#define CACHEIR_B200_DENSE_F32 1         /* y as float32                                             */
#define CACHEIR_B200_DENSE_SILU 2        /* silu on columns [0, act_cols), the rest unchanged        */
#define CACHEIR_B200_DENSE_GEGLU 3       /* W rows alternate gate, up; gelu_tanh(gate) * up, [T, N/2] */
#define CACHEIR_B200_DENSE_GATED 4       /* y * sigmoid(gate[t, column])                             */
#define CACHEIR_B200_DENSE_RESIDUAL 5    /* residual += tanh(norm_alpha * y) * norm_w + norm_b, then next_mode */
#define CACHEIR_B200_DENSE_GELU_EMBED 6  /* gelu_tanh(y) * table[ids[t], table_col + column]         */

typedef struct {
  const void* x;            /* bf16 [T, x_stride]                                        */
  const void* w;            /* bf16 [N, w_stride]; batch > 1: entry z starts at row z*w_batch_rows */
  void* y;
  int T, N, K, batch;
  int w_batch_rows, x_batch_cols, y_batch_cols, epilogue;
  long long w_stride, x_stride, y_stride;
  int act_cols, next_mode, vocab, table_col;
  const void* gate;         /* bf16 [T, gate_stride], indexed by output column */
  long long gate_stride;
  float* residual;          /* [T, N] */
  const float* norm_w;
  const float* norm_b;
  const float* next_w;
  const float* next_b;
  void* next_out;           /* bf16 [T, N] */
  float norm_alpha, next_alpha;
  const int64_t* ids;
  const void* table;        /* bf16 [vocab, table_stride] */
  long long table_stride;
} cacheir_b200_dense_args;

/* Tensor-core GEMM Y = f(X W^T), bf16 operands. Strides must be multiples of 8 elements. */
int cacheir_b200_dense_supported(int K, long long w_stride, long long x_stride, int batch, int x_batch_cols);
int cacheir_b200_dense_gemm(const cacheir_b200_dense_args* args, void* stream);

/* The same product on the CUDA cores in true float32 arithmetic, any extents; y has type y_dtype. */
int cacheir_b200_dense_simple(const void* x, const void* w, void* y, int T, int N, int K, int batch, int w_batch_rows,
                              int x_batch_cols, int y_batch_cols, long long w_stride, long long x_stride, long long y_stride,
                              int dtype, int y_dtype, void* stream);

/* residual = table[ids] * scale, then next_mode. `table` and `next_out` are of `dtype`. */
int cacheir_b200_scaled_embedding(const void* table, const int64_t* ids, float* residual, int rows, int width, int vocab,
                                  float scale, int next_mode, const float* next_w, const float* next_b, float next_alpha,
                                  void* next_out, int dtype, void* stream);
/* out[j] = dyt(residual[row_index ? row_index[j] : j]) */
int cacheir_b200_dyt_rows(const float* residual, const int32_t* row_index, const float* w, const float* b, float alpha, void* out,
                          int rows, int width, int dtype, void* stream);
/* residual += dyt(y), then next_mode */
int cacheir_b200_residual_dyt(float* residual, const void* y, const float* w, const float* b, float alpha, int rows, int width,
                              int next_mode, const float* next_w, const float* next_b, float next_alpha, void* next_out,
                              int dtype, void* stream);
/* residual += y / sqrt(mean(y^2) + eps) * w, then next_mode */
int cacheir_b200_residual_rms(float* residual, const void* y, const float* w, float eps, int rows, int width, int next_mode,
                              const float* next_w, const float* next_b, float next_alpha, void* next_out, int dtype, void* stream);
/* out = o / sqrt(mean(o^2) + eps) * w * sigmoid(gate) */
int cacheir_b200_gated_rms(const void* o, const void* gate, long long gate_stride, const float* w, float eps, void* out, int rows,
                           int cols, int dtype, void* stream);
/* y [rows, 2*ff], columns alternating gate, up -> out [rows, ff] = gelu_tanh(gate) * up */
int cacheir_b200_geglu_pairs(const void* y, void* out, int rows, int ff, int dtype, void* stream);
/* out = gelu_tanh(g) * table[ids, table_col + column] */
int cacheir_b200_gelu_embed(const void* g, const int64_t* ids, const void* table, long long table_stride, int table_col, void* out,
                            int rows, int dim, int vocab, int dtype, void* stream);
/* silu in place on columns [0, cols) of y [rows, stride] */
int cacheir_b200_silu_cols(void* y, int rows, long long stride, int cols, int dtype, void* stream);

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

/* ---- linear recurrence S <- decay S + k v^T, o = S^T q, one float32 state [heads, dim, vdim] per slot ------------- */
typedef struct {
  const int32_t* positions;
  const int32_t* cu_rows;
  const int32_t* slots;
  int rows, segments;
  int heads, dim, vdim;
  const void* q;            /* [rows, stride], heads*dim columns, activation already applied */
  const void* k;
  const void* v;            /* heads*vdim columns */
  long long stride;         /* common row stride of q, k, v */
  const float* decay_pow;   /* [heads, 65]: decay^0 .. decay^64 */
  float* state;             /* [num_slots, heads, dim, vdim] */
  int num_slots;
  void* out;                /* [rows, heads*vdim] */
  int dtype;
} cacheir_b200_recurrence_args;

/* Token by token, any extents. A sequence whose first row has position 0 starts from a zero state. */
int cacheir_b200_recurrence_simple(const cacheir_b200_recurrence_args* a, void* stream);
/* One row per segment, streaming the state once (vdim % 4 == 0, otherwise EUNSUPPORTED). */
int cacheir_b200_recurrence_step(const cacheir_b200_recurrence_args* a, void* stream);
/* Chunked tensor-core form (bf16 q, k, v; dim % 16 == 0, dim <= 128, vdim % 8 == 0). Sequences longer than 256 rows use the
 * workspace for the states between their 256-row parts. */
int cacheir_b200_recurrence_chunked_supported(int dim, int vdim, int dtype);
size_t cacheir_b200_recurrence_workspace_bytes(int rows, int segments, int heads, int dim, int vdim);
int cacheir_b200_recurrence_chunked(const cacheir_b200_recurrence_args* a, void* workspace, size_t workspace_bytes, void* stream);

/* First bounded wait of this library's kernels that gave up since the last reset (0: none). Synchronises. */
int cacheir_b200_hybrid_device_status(int reset);

#ifdef __cplusplus
}
#endif
#endif
