// One block finishes a row of the 32-bit residual stream and leaves the next operator's input: the row itself, its RMS norm or
// its layer norm.
#pragma once

#include "hybrid_common.cuh"

namespace cb200 {

struct RowNext {
  int mode;             // NEXT_NONE, NEXT_COPY, NEXT_RMS or NEXT_LAYER
  const float* w;
  float eps;
  void* out;
};

inline bool row_next_norms(int mode) { return mode == CACHEIR_B200_NEXT_RMS || mode == CACHEIR_B200_NEXT_LAYER; }
inline bool row_next_ok(int mode, const float* w, const void* out) {
  return mode == CACHEIR_B200_NEXT_NONE || (mode == CACHEIR_B200_NEXT_COPY && out) || (row_next_norms(mode) && w && out);
}
inline bool row_next_aligned(int mode, const float* w, const void* out) {
  return mode == CACHEIR_B200_NEXT_NONE || (aligned_to(out, 16) && (!row_next_norms(mode) || aligned_to(w, 16)));
}

// value(c, s): the row's new entries c .. c + VEC - 1 from their old ones in s. A thread reads and writes the same columns
// throughout, so `nx.out` may be what `value` reads.
template <typename T, int VEC, typename Value>
__device__ __forceinline__ void finish_row(float* xr, size_t row, int width, const RowNext& nx, float* scratch, Value value) {
  T* out = static_cast<T*>(nx.out) + row * width;
  const int step = static_cast<int>(blockDim.x) * VEC;
  const bool centred = nx.mode == CACHEIR_B200_NEXT_LAYER;
  float ss = 0.f;                      // of squares, or of the entries
  for (int c = threadIdx.x * VEC; c < width; c += step) {
    float s[VEC];
    load_vec<float, VEC>(xr + c, s);
    value(c, s);
    store_vec<float, VEC>(xr + c, s);
    if (nx.mode == CACHEIR_B200_NEXT_COPY) store_vec<T, VEC>(out + c, s);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = centred ? ss + s[i] : fmaf(s[i], s[i], ss);
  }
  if (nx.mode != CACHEIR_B200_NEXT_RMS && !centred) return;
  float mean = 0.f;
  if (centred) {
    mean = block_sum_all(ss, scratch) / static_cast<float>(width);
    ss = 0.f;
    for (int c = threadIdx.x * VEC; c < width; c += step) {
      float s[VEC];
      load_vec<float, VEC>(xr + c, s);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(s[i] - mean, s[i] - mean, ss);
    }
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, scratch) / static_cast<float>(width) + nx.eps);
  for (int c = threadIdx.x * VEC; c < width; c += step) {
    float s[VEC], w[VEC];
    load_vec<float, VEC>(xr + c, s);
    load_vec<float, VEC>(nx.w + c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) s[i] = (s[i] - mean) * inv * w[i];
    store_vec<T, VEC>(out + c, s);
  }
}

}  // namespace cb200
