/*
 * cacheir_b200_recurrence.h -- C ABI of libcacheir_b200_recurrence.so: linear recurrences (Gutorax), matrix memory
 * (Rekodra) and state spaces (Zimorax). Rows of a step as in cacheir_b200_ragged.h.
 */
#ifndef CACHEIR_B200_RECURRENCE_H_
#define CACHEIR_B200_RECURRENCE_H_

#include "cacheir_b200_ragged.h"

#ifdef __cplusplus
extern "C" {
#endif

/* ---- linear recurrence S <- decay S + take k v^T, o = S^T q, one float32 state [heads, dim, vdim] per slot -----------
 * Constant decays (decay_pow): take is one. Gated (decay_pow NULL): logarithms of both per token and head; with a `normaliser`
 * behind a slot's state lie n [heads, dim], which follows n <- decay n + take k, and [heads] running maxima
 * (cacheir_b200_memory_gates). Neighbouring heads may share queries and keys (key_heads); with `skip`, o += skip[head] * v. */
typedef struct {
  const int32_t* positions;
  const int32_t* cu_rows;
  const int32_t* slots;
  int rows, segments;
  int heads, dim, vdim;
  const void* q;            /* [rows, stride], key_heads*dim columns, activation already applied */
  const void* k;
  const void* v;            /* heads*vdim columns */
  long long stride;         /* common row stride of q, k, v */
  const float* decay_pow;   /* [heads, 65]: decay^0 .. decay^64 */
  float* state;             /* slot s at s * slot_stride */
  int num_slots;
  void* out;                /* [rows, heads*vdim] */
  int dtype;
  long long slot_stride;    /* floats from slot to slot */
  /* gated form */
  const float* log_decay;   /* [rows, heads] */
  const float* log_take;
  float* normaliser;        /* [rows, heads]: q . n; NULL: there is no n */
  float q_scale;            /* q is multiplied with it */
  int key_heads;            /* 0: heads */
  const float* skip;        /* [heads] or NULL */
} cacheir_b200_recurrence_args;

/* Token by token, any extents. A sequence whose first row has position 0 starts from a zero state. */
int cacheir_b200_recurrence_simple(const cacheir_b200_recurrence_args* a, void* stream);
/* One row per segment, constant decays, streaming the state once (vdim % 4 == 0, otherwise EUNSUPPORTED). */
int cacheir_b200_recurrence_step(const cacheir_b200_recurrence_args* a, void* stream);
/* Chunked tensor-core form (bf16 q, k, v; dim % 16 == 0, dim <= 128, vdim % 8 == 0). Sequences longer than 256 rows use the
 * workspace for the states between their 256-row parts. */
int cacheir_b200_recurrence_chunked_supported(int dim, int vdim, int dtype);
size_t cacheir_b200_recurrence_workspace_bytes(int rows, int segments, int heads, int dim, int vdim);
int cacheir_b200_recurrence_chunked(const cacheir_b200_recurrence_args* a, void* workspace, size_t workspace_bytes, void* stream);

/* ---- matrix memory: a gated recurrence whose sums are divided by a normaliser -------------------------------------------
 * logits [rows, stride]: input gates of all heads, then forget gates. i = cap tanh((z + bias) / cap) likewise for the forget
 * gate, f = log sigmoid of it; m <- max(f + m, i) starting from 0; log decay = f + m_before - m, log take = i - m. */
int cacheir_b200_memory_gates(const cacheir_b200_recurrence_args* a, const float* logits, long long stride, const float* in_bias,
                              const float* forget_bias, float cap, float* log_decay, float* log_take, float* maximum, void* stream);
/* out = x / rms(x) * w * sigmoid(gate) per head, x = o / (max(|normaliser|, exp(-maximum)) + 1e-6); w [heads*vdim] */
int cacheir_b200_memory_norm(const void* o, const float* normaliser, const float* maximum, const void* gate, long long gate_stride,
                             const float* w, float eps, void* out, int rows, int heads, int vdim, int dtype, void* stream);
/* Gates, one token of the recurrence, and the norm: one row per segment (vdim % 4 == 0, otherwise EUNSUPPORTED). */
int cacheir_b200_memory_step(const cacheir_b200_recurrence_args* a, const float* logits, long long stride, const float* in_bias,
                             const float* forget_bias, float cap, const void* gate, long long gate_stride, const float* w, float eps,
                             void* stream);

/* ---- state space: a gated recurrence with log decay -exp(log_rate) dt and take dt, dt = softplus(z + bias) -----------------
 * z [rows, stride] with a column per head; bias and log_rate [heads]. */
int cacheir_b200_state_space_gates(const cacheir_b200_recurrence_args* a, const float* z, long long stride, const float* bias,
                                   const float* log_rate, float* log_decay, float* log_take, void* stream);
/* Gates and one token of the recurrence: one row per segment (vdim % 4 == 0, otherwise EUNSUPPORTED). */
int cacheir_b200_state_space_step(const cacheir_b200_recurrence_args* a, const float* z, long long stride, const float* bias,
                                  const float* log_rate, void* stream);

/* Always 0: these kernels wait for nothing. */
int cacheir_b200_recurrence_device_status(int reset);

#ifdef __cplusplus
}
#endif
#endif
