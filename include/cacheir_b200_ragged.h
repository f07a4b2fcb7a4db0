/*
 * cacheir_b200_ragged.h -- C ABI of libcacheir_b200_ragged.so: the dense products and row operators that every family
 * with ragged steps uses (beside it lies the library of the family's own mixers). Conventions are those of
 * cacheir_b200.h: device pointers and sizes only, no allocation, no synchronisation, 0 / positive cudaError_t / negative
 * CACHEIR_B200_E* return values.
 *
 * A step runs `rows` token rows of `segments` sequences. Rows of one sequence are neighbours in position order:
 *   cu_rows   [segments + 1]  first row of every sequence (cu_rows[segments] = rows in use; later rows are padding)
 *   row_seg   [rows]          sequence of a row, -1 for padding
 *   positions [rows]          position of a row in its sequence
 *   page_table [segments, max_pages], slots [segments]: where the sequence's cache pages and recurrent state live
 * The residual stream is float32; activations are `dtype` (F32 or BF16); norm weights are float32.
 */
#ifndef CACHEIR_B200_RAGGED_H_
#define CACHEIR_B200_RAGGED_H_

#include "cacheir_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

/* What a kernel that finishes the residual stream leaves as the next operator's input */
#define CACHEIR_B200_NEXT_NONE 0
#define CACHEIR_B200_NEXT_COPY 1   /* the residual itself, rounded to the activation type */
#define CACHEIR_B200_NEXT_DYT 2    /* tanh(alpha * residual) * w + b                      */
#define CACHEIR_B200_NEXT_RMS 3    /* residual / sqrt(mean(residual^2) + alpha) * w       */
#define CACHEIR_B200_NEXT_LAYER 4  /* (residual - mean) / sqrt(variance + alpha) * w      */

/* Epilogues of cacheir_b200_dense_gemm */
#define CACHEIR_B200_DENSE_BF16 0        /* y                                                        */
#define CACHEIR_B200_DENSE_F32 1         /* y as float32                                             */
#define CACHEIR_B200_DENSE_SILU 2        /* silu on columns [0, act_cols), the rest unchanged        */
#define CACHEIR_B200_DENSE_GEGLU 3       /* W rows alternate gate, up; gelu_tanh(gate) * up, [T, N/2] */
#define CACHEIR_B200_DENSE_GATED 4       /* y * sigmoid(gate[t, column])                             */
#define CACHEIR_B200_DENSE_RESIDUAL 5    /* residual += tanh(norm_alpha * y) * norm_w + norm_b, then next_mode */
#define CACHEIR_B200_DENSE_GELU_EMBED 6  /* gelu_tanh(y) * table[ids[t], table_col + column]         */
#define CACHEIR_B200_DENSE_SWIGLU 7      /* as GEGLU with silu(gate) * up                            */
#define CACHEIR_B200_DENSE_CLAMPED_GLU 8 /* as GEGLU with g sigmoid(1.702 g) (u + 1), g = min(gate, limit), u = up in [-limit, limit] */
#define CACHEIR_B200_DENSE_RELU2 9       /* max(y, 0)^2 */

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
  const float* bias;        /* [N] added to y before the epilogue, or NULL (batch 1) */
  float limit;
  int tail_cols;            /* BF16, SILU and the paired epilogues: the last tail_cols columns of y go to `tail` as float32 instead */
  float* tail;              /* [T, tail_stride] */
  long long tail_stride;
} cacheir_b200_dense_args;

/* Tensor-core GEMM Y = f(X W^T), bf16 operands. Strides must be multiples of 8 elements. */
int cacheir_b200_dense_supported(int K, long long w_stride, long long x_stride, int batch, int x_batch_cols);
int cacheir_b200_dense_gemm(const cacheir_b200_dense_args* args, void* stream);

/* The same product on the CUDA cores in true float32 arithmetic, any extents; y has type y_dtype. */
int cacheir_b200_dense_simple(const void* x, const void* w, void* y, int T, int N, int K, int batch, int w_batch_rows,
                              int x_batch_cols, int y_batch_cols, long long w_stride, long long x_stride, long long y_stride,
                              const float* bias, int dtype, int y_dtype, void* stream);

/* residual = table[ids] * scale (`accumulate`: +=), then next_mode. `table` and `next_out` are of `dtype`. */
int cacheir_b200_scaled_embedding(const void* table, const int64_t* ids, float* residual, int rows, int width, int vocab,
                                  float scale, int accumulate, int next_mode, const float* next_w, const float* next_b, float next_alpha,
                                  void* next_out, int dtype, void* stream);
/* out[j] = dyt(residual[row_index ? row_index[j] : j]) */
int cacheir_b200_dyt_rows(const float* residual, const int32_t* row_index, const float* w, const float* b, float alpha, void* out,
                          int rows, int width, int dtype, void* stream);
/* out[j] = x / sqrt(mean(x^2) + eps) * w, x = residual[row_index ? row_index[j] : j] */
int cacheir_b200_rms_rows(const float* residual, const int32_t* row_index, const float* w, float eps, void* out, int rows, int width,
                          int dtype, void* stream);
/* out[j] = (x - mean) / sqrt(variance + eps) * w, x = residual[row_index ? row_index[j] : j] */
int cacheir_b200_layer_norm_rows(const float* residual, const int32_t* row_index, const float* w, float eps, void* out, int rows,
                                 int width, int dtype, void* stream);
/* out [rows, 2*width] = (residual | table[ids]), the input of a product that meets the embedding output again */
int cacheir_b200_join_embedding(const float* residual, const void* table, const int64_t* ids, void* out, int rows, int width, int vocab,
                                int dtype, void* stream);
/* residual += y * scale (scale [width], NULL: ones), then next_mode (NONE, COPY, RMS or LAYER) */
int cacheir_b200_residual_add(float* residual, const void* y, const float* scale, int rows, int width, int next_mode, const float* next_w, const float* next_b,
                              float next_alpha, void* next_out, int dtype, void* stream);
/* residual += factor * (rms(y1) * w1 + rms(y2) * w2) with rms(y) = y / sqrt(mean(y^2) + eps), then next_mode (NONE, COPY or RMS) */
int cacheir_b200_residual_rms_pair(float* residual, const void* y1, const float* w1, const void* y2, const float* w2, float factor, float eps,
                                   int rows, int width, int next_mode, const float* next_w, const float* next_b, float next_alpha,
                                   void* next_out, int dtype, void* stream);
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
/* y [rows, 2*ff], columns alternating gate, up -> out [rows, ff] as the paired epilogue `epilogue` leaves it */
int cacheir_b200_glu_pairs(const void* y, void* out, int rows, int ff, int epilogue, float limit, int dtype, void* stream);
/* out = gelu_tanh(g) * table[ids, table_col + column] */
int cacheir_b200_gelu_embed(const void* g, const int64_t* ids, const void* table, long long table_stride, int table_col, void* out,
                            int rows, int dim, int vocab, int dtype, void* stream);
/* silu in place on columns [0, cols) of y [rows, stride]; likewise max(y, 0)^2 */
int cacheir_b200_silu_cols(void* y, int rows, long long stride, int cols, int dtype, void* stream);
int cacheir_b200_relu2_cols(void* y, int rows, long long stride, int cols, int dtype, void* stream);
/* Norm in `parts` equal parts of a row, each by its own root mean square, with a gate [rows, gate_stride] and a weight w (one entry
 * per column, or with shared_weight per column of a part):
 *   gate_first:  y = o * silu(gate), out = y / sqrt(mean(y^2) + eps) * w        else  out = o / sqrt(mean(o^2) + eps) * w * silu(gate) */
int cacheir_b200_gated_parts_rms(const void* o, const void* gate, long long gate_stride, const float* w, int shared_weight, int gate_first,
                                 float eps, void* out, int rows, int cols, int parts, int dtype, void* stream);

/* First bounded wait of this library's kernels that gave up since the last reset (0: none). Synchronises. */
int cacheir_b200_ragged_device_status(int reset);

#ifdef __cplusplus
}
#endif
#endif
