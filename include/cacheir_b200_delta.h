/*
 * cacheir_b200_delta.h -- C ABI of libcacheir_b200_delta.so: short causal convolutions with carried inputs, and the gated delta
 * rule (Zimorax). Rows of a step as in cacheir_b200_ragged.h.
 */
#ifndef CACHEIR_B200_DELTA_H_
#define CACHEIR_B200_DELTA_H_

#include "cacheir_b200_ragged.h"

#ifdef __cplusplus
extern "C" {
#endif

/* ---- short convolution: y[t] = silu(sum_j w[channel, j] x[t - (taps - 1) + j] + bias), zeros before position 0 -------------
 * A sequence's last taps - 1 inputs lie in its slot as float32 [taps - 1, channels] (oldest first). */
typedef struct {
  const int32_t* positions;
  const int32_t* cu_rows;
  const int32_t* slots;
  int rows, segments, channels, taps;
  const void* x;            /* [rows, stride] */
  long long stride;
  const float* w;           /* [channels, taps], the current token's last */
  const float* bias;        /* [channels] or NULL */
  float* state;             /* slot s at s * slot_stride */
  long long slot_stride;
  int num_slots, dtype;
  void* out;                /* [rows, out_stride] */
  long long out_stride;
} cacheir_b200_conv_args;
int cacheir_b200_short_conv(const cacheir_b200_conv_args* a, void* stream);

/* ---- gated delta rule, one float32 state [heads, dim, vdim] per slot ------------------------------------------------------
 *   S <- decay S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
 * k and q are the given rows divided by sqrt(sum of squares + 1e-6), q also times dim^(-1/2); neighbouring heads share them.
 * beta = sigmoid(zb), decay = exp(-exp(log_rate) softplus(za + bias)), z [rows, z_stride] = (zb of all heads | za of all heads). */
typedef struct {
  const int32_t* positions;
  const int32_t* cu_rows;
  const int32_t* slots;
  int rows, segments, heads, key_heads, dim, vdim;
  const void* q;            /* [rows, stride], key_heads*dim columns */
  const void* k;
  const void* v;            /* heads*vdim columns */
  long long stride;
  const float* z;
  long long z_stride;
  const float* bias;        /* [heads] */
  const float* log_rate;    /* [heads] */
  float* state;
  long long slot_stride;
  int num_slots, dtype;
  void* out;                /* [rows, heads*vdim] */
} cacheir_b200_delta_args;

/* Token by token, any extents. A sequence whose first row has position 0 starts from a zero state. */
int cacheir_b200_delta_simple(const cacheir_b200_delta_args* a, void* stream);
/* One row per segment; out = o / sqrt(mean(o^2) + eps) * w * silu(gate) per head, w [vdim] shared by the heads, gate [rows,
 * gate_stride] (vdim % 4 == 0 and vdim <= 1024, otherwise EUNSUPPORTED). */
int cacheir_b200_delta_step(const cacheir_b200_delta_args* a, const void* gate, long long gate_stride, const float* w, float eps, void* stream);
/* Chunked tensor-core form (bf16; dim % 16 == 0, dim <= 128, vdim % 8 == 0), 64 tokens at a time. */
int cacheir_b200_delta_chunked_supported(int dim, int vdim, int dtype);
size_t cacheir_b200_delta_workspace_bytes(int rows, int segments, int heads);
int cacheir_b200_delta_chunked(const cacheir_b200_delta_args* a, void* workspace, size_t workspace_bytes, void* stream);

/* Always 0: these kernels wait for nothing. */
int cacheir_b200_delta_device_status(int reset);

#ifdef __cplusplus
}
#endif
#endif
