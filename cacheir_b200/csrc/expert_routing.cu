// Around the experts' products: which tokens go to which expert, and the weighted sum of what comes back with the
// sublayer's RMS norm and residual add.
#include "cacheir_b200_experts.h"
#include "hybrid_common.cuh"

namespace cb200 {
namespace {

constexpr int kRouteThreads = 256;      // a warp per token

// Every block chooses for its tokens and counts; the block that finishes last turns counts into places (nobody waits).
__global__ void __launch_bounds__(kRouteThreads)
route_kernel(const float* __restrict__ logits, long long stride, const int32_t* __restrict__ row_seg, int rows, int experts, int top,
             float scale, int32_t* counters, int32_t* __restrict__ cu, int32_t* __restrict__ token_of, int32_t* place_of,
             float* __restrict__ weight, int32_t* chosen) {
  extern __shared__ int s_first[];      // [experts + 1]
  __shared__ int s_sum[kRouteThreads / 32];
  __shared__ bool s_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = blockIdx.x * (kRouteThreads / 32) + warp;
  if (row < rows) {
    const float* z = logits + static_cast<long long>(row) * stride;
    const bool real = row_seg[row] >= 0;
    float bound = INFINITY;             // the last choice: what follows it in (value descending, index ascending) order is next
    int after = -1;
    for (int k = 0; k < top; ++k) {
      float best = -INFINITY;
      int at = experts;
      for (int e = lane; e < experts; e += 32) {
        const float v = z[e];
        if ((v < bound || (v == bound && e > after)) && (v > best || at == experts)) { best = v; at = e; }
      }
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, best, off);
        const int e = __shfl_xor_sync(0xffffffffu, at, off);
        if (e < experts && (at == experts || v > best || (v == best && e < at))) { best = v; at = e; }
      }
      bound = best;
      after = at;
      if (lane == 0) {
        const bool take = real && at < experts;      // (a row of NaNs chooses nothing)
        chosen[row * top + k] = take ? at : -1;
        weight[row * top + k] = take ? sigmoid_exact(best) * scale : 0.f;
        place_of[row * top + k] = take ? atomicAdd(&counters[at], 1) : -1;      // its rank within the expert, for now
      }
    }
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(&counters[experts], 1) == static_cast<int>(gridDim.x) - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  int base = 0;
  for (int e0 = 0; e0 < experts; e0 += kRouteThreads) {      // exclusive prefix sums of the counts
    const int e = e0 + static_cast<int>(threadIdx.x);
    const int n = e < experts ? __ldcg(&counters[e]) : 0;
    int incl = n;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, incl, off);
      if (lane >= off) incl += up;
    }
    if (lane == 31) s_sum[warp] = incl;
    __syncthreads();
    int before = base, total = 0;
    for (int w = 0; w < kRouteThreads / 32; ++w) {
      if (w < warp) before += s_sum[w];
      total += s_sum[w];
    }
    if (e < experts) {
      s_first[e] = before + incl - n;
      cu[e] = before + incl - n;
      counters[e] = 0;
    }
    base += total;
    __syncthreads();
  }
  if (threadIdx.x == 0) {
    cu[experts] = base;
    counters[experts] = 0;
  }
  for (int i = threadIdx.x; i < rows * top; i += kRouteThreads) {
    const int e = __ldcg(&chosen[i]);
    if (e < 0) continue;
    const int place = s_first[e] + __ldcg(&place_of[i]);
    place_of[i] = place;
    token_of[place] = i / top;
  }
}

// SAVED: the sums stay in shared memory between the two passes
template <typename T, int VEC, bool SAVED>
__global__ void __launch_bounds__(512)
combine_kernel(float* __restrict__ x, const T* __restrict__ y, const int32_t* __restrict__ place_of, const float* __restrict__ weight, int top,
               const T* __restrict__ shared, const float* __restrict__ w, float eps, int width, T* next_out) {
  extern __shared__ float s_m[];
  __shared__ float scratch[32];
  const size_t row = blockIdx.x;
  auto mixed = [&](int c, float (&m)[VEC]) {
    if (shared) {
      load_vec<T, VEC>(shared + row * width + c, m);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) m[i] = 0.f;
    }
    for (int k = 0; k < top; ++k) {
      const int place = place_of[row * top + k];
      if (place < 0) continue;
      const float a = weight[row * top + k];
      float v[VEC];
      load_vec<T, VEC>(y + static_cast<size_t>(place) * width + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) m[i] = fmaf(a, v[i], m[i]);
    }
  };
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < width; c += 512 * VEC) {
    float m[VEC];
    mixed(c, m);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(m[i], m[i], ss);
    if (SAVED) store_vec<float, VEC>(s_m + c, m);
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, scratch) / static_cast<float>(width) + eps);
  for (int c = threadIdx.x * VEC; c < width; c += 512 * VEC) {
    float m[VEC], wv[VEC], s[VEC];
    if (SAVED) load_vec<float, VEC>(s_m + c, m);
    else mixed(c, m);
    load_vec<float, VEC>(w + c, wv);
    load_vec<float, VEC>(x + row * width + c, s);
#pragma unroll
    for (int i = 0; i < VEC; ++i) s[i] = fmaf(m[i] * inv, wv[i], s[i]);
    store_vec<float, VEC>(x + row * width + c, s);
    if (next_out) store_vec<T, VEC>(next_out + row * width + c, s);
  }
}

}  // namespace
}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_route(const float* logits, long long stride, const int32_t* row_seg, int rows, int experts, int top, float scale,
                                  int32_t* counters, int32_t* cu, int32_t* token_of, int32_t* place_of, float* weight, int32_t* chosen,
                                  void* stream) {
  if (rows <= 0) return 0;
  if (!logits || !row_seg || experts < 1 || top < 1 || top > experts || stride < experts || !counters || !cu || !token_of || !place_of ||
      !weight || !chosen)
    return CACHEIR_B200_EINVAL;
  const size_t smem = static_cast<size_t>(experts + 1) * 4;
  if (smem > 40 * 1024) return CACHEIR_B200_ELIMIT;
  route_kernel<<<(rows + 7) / 8, kRouteThreads, smem, as_stream(stream)>>>(logits, stride, row_seg, rows, experts, top, scale, counters, cu,
                                                                          token_of, place_of, weight, chosen);
  return launch_status();
}

extern "C" int cacheir_b200_combine_residual_rms(float* residual, const void* y, const int32_t* place_of, const float* weight, int top,
                                                 const void* shared, const float* w, float eps, int rows, int width, int next_mode,
                                                 void* next_out, int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !y || !place_of || !weight || top < 1 || !w || (next_mode != CACHEIR_B200_NEXT_NONE && next_mode != CACHEIR_B200_NEXT_COPY) ||
      (next_mode == CACHEIR_B200_NEXT_COPY && !next_out))
    return CACHEIR_B200_EINVAL;
  void* out = next_mode == CACHEIR_B200_NEXT_COPY ? next_out : nullptr;
  const bool vec = width % 4 == 0 && aligned_to(residual, 16) && aligned_to(y, 16) && aligned_to(w, 16) && aligned_to(shared, 16) && aligned_to(out, 16);
  const bool saved = width <= 11 * 1024;
  const size_t smem = saved ? static_cast<size_t>(width) * 4 : 0;
#define CB200_COMBINE(VEC, SAVED)                                                                                              \
  combine_kernel<T, VEC, SAVED><<<rows, 512, smem, as_stream(stream)>>>(residual, static_cast<const T*>(y), place_of, weight, top, \
                                                                       static_cast<const T*>(shared), w, eps, width, static_cast<T*>(out))
  CB200_HYBRID_DTYPE(dtype, {
    if (vec && saved) CB200_COMBINE(4, true);
    else if (vec) CB200_COMBINE(4, false);
    else if (saved) CB200_COMBINE(1, true);
    else CB200_COMBINE(1, false);
  });
#undef CB200_COMBINE
  return launch_status();
}
