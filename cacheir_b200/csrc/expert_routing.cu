// Around the experts' products: which tokens go to which expert, and the weighted sum of what comes back with the
// sublayer's RMS norm and residual add.
#include "cacheir_b200_experts.h"
#include "hybrid_common.cuh"

namespace cb200 {
namespace {

constexpr int kRouteThreads = 256;      // a warp per token
constexpr int kHeld = 4;                // logits a lane keeps in registers

// The warp's token: its choices in order, each with its rank among the tokens of that expert (in no particular order).
template <bool HELD>
__device__ __forceinline__ void choose(const float* z, bool real, int row, int experts, int top, float scale, int32_t* counters,
                                       int32_t* place_of, float* weight, int32_t* chosen) {
  const int lane = threadIdx.x & 31;
  float held[kHeld];
  if (HELD) {
#pragma unroll
    for (int i = 0; i < kHeld; ++i) held[i] = lane + 32 * i < experts ? z[lane + 32 * i] : 0.f;
  }
  float bound = INFINITY;               // the last choice: what follows it in (value descending, index ascending) order is next
  int after = -1, mine = -1;
  float mine_z = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = experts;
    auto look = [&](int e, float v) {
      if ((v < bound || (v == bound && e > after)) && (v > best || at == experts)) { best = v; at = e; }
    };
    if (HELD) {
#pragma unroll
      for (int i = 0; i < kHeld; ++i)
        if (lane + 32 * i < experts) look(lane + 32 * i, held[i]);
    } else {
      for (int e = lane; e < experts; e += 32) look(e, z[e]);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
      const float v = __shfl_xor_sync(0xffffffffu, best, off);
      const int e = __shfl_xor_sync(0xffffffffu, at, off);
      if (e < experts && (at == experts || v > best || (v == best && e < at))) { best = v; at = e; }
    }
    bound = best;
    after = at;
    if (lane == k % 32) { mine = at; mine_z = best; }
    if (k % 32 == 31 || k == top - 1) { // the lanes record what they hold: one round of atomics for up to 32 choices
      const int j = k / 32 * 32 + lane;
      if (j <= k) {
        const bool take = real && mine < experts;      // (a row of NaNs chooses nothing)
        chosen[row * top + j] = take ? mine : -1;
        weight[row * top + j] = take ? sigmoid_exact(mine_z) * scale : 0.f;
        place_of[row * top + j] = take ? atomicAdd(&counters[mine], 1) : -1;
      }
    }
  }
}

// Every block chooses for its tokens and counts; the block that finishes last turns counts into places (nobody waits).
// PLACE false: choices and ranks only.
template <bool HELD, bool PLACE>
__global__ void __launch_bounds__(kRouteThreads)
route_kernel(const float* __restrict__ logits, long long stride, const int32_t* __restrict__ row_seg, int rows, int experts, int top,
             float scale, int32_t* counters, int32_t* __restrict__ cu, int32_t* __restrict__ token_of, int32_t* place_of,
             float* __restrict__ weight, int32_t* chosen) {
  extern __shared__ int s_first[];      // [experts + 1]
  __shared__ int s_sum[kRouteThreads / 32];
  __shared__ bool s_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = blockIdx.x * (kRouteThreads / 32) + warp;
  if (row < rows)
    choose<HELD>(logits + static_cast<long long>(row) * stride, row_seg[row] >= 0, row, experts, top, scale, counters, place_of, weight, chosen);
  if (!PLACE) return;
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
    const int e = __ldcg(&chosen[i]), rank = __ldcg(&place_of[i]);
    if (e < 0) continue;
    const int place = s_first[e] + rank;
    place_of[i] = place;
    token_of[place] = i / top;
  }
}

// Places from ranks, and every row's copy at each of its places: a block per row, each adding up the counts it needs.
__global__ void __launch_bounds__(kRouteThreads)
place_kernel(int rows, int experts, int top, int32_t* counters, int32_t* __restrict__ cu, int32_t* __restrict__ token_of,
             int32_t* __restrict__ place_of, const int32_t* __restrict__ chosen, const uint4* __restrict__ x, uint4* __restrict__ placed,
             int pieces) {
  extern __shared__ int s_count[];      // [experts], then [top] places
  __shared__ bool s_last;
  int* s_place = s_count + experts;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x;
  for (int e = threadIdx.x; e < experts; e += kRouteThreads) s_count[e] = __ldcg(&counters[e]);
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(&counters[experts], 1) == static_cast<int>(gridDim.x) - 1;
  for (int k = warp; k < top; k += kRouteThreads / 32) {
    const int e = chosen[row * top + k];
    int before = 0;
    for (int i = lane; i < e; i += 32) before += s_count[i];
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) before += __shfl_xor_sync(0xffffffffu, before, off);
    if (lane == 0) {
      const int place = e < 0 ? -1 : before + place_of[row * top + k];
      s_place[k] = place;
      if (e >= 0) {
        place_of[row * top + k] = place;
        token_of[place] = row;
      }
    }
  }
  __syncthreads();
  for (int c = threadIdx.x; c < pieces; c += kRouteThreads) {
    const uint4 v = x[static_cast<size_t>(row) * pieces + c];
    for (int k = 0; k < top; ++k)
      if (s_place[k] >= 0) placed[static_cast<size_t>(s_place[k]) * pieces + c] = v;
  }
  if (s_last) {                         // every block has read the counts
    if (threadIdx.x == 0) {
      int at = 0;
      for (int e = 0; e < experts; ++e) {
        cu[e] = at;
        at += s_count[e];
      }
      cu[experts] = at;
    }
    for (int e = threadIdx.x; e <= experts; e += kRouteThreads) counters[e] = 0;
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
                                  const void* x, void* placed, int row_bytes, void* stream) {
  if (rows <= 0) return 0;
  if (!logits || !row_seg || experts < 1 || top < 1 || top > experts || stride < experts || !counters || !cu || !token_of || !place_of ||
      !weight || !chosen || (placed && (!x || row_bytes <= 0)))
    return CACHEIR_B200_EINVAL;
  if (placed && (row_bytes % 16 != 0 || !aligned_to(x, 16) || !aligned_to(placed, 16))) return CACHEIR_B200_EALIGN;
  const size_t smem = static_cast<size_t>(experts + top + 1) * 4;
  if (smem > 40 * 1024) return CACHEIR_B200_ELIMIT;
  const int blocks = (rows + 7) / 8;
  cudaStream_t st = as_stream(stream);
#define CB200_ROUTE(HELD, PLACE)                                                                                                    \
  route_kernel<HELD, PLACE><<<blocks, kRouteThreads, PLACE ? smem : 0, st>>>(logits, stride, row_seg, rows, experts, top, scale, counters, \
                                                                             cu, token_of, place_of, weight, chosen)
  if (!placed) {
    if (experts <= 32 * kHeld) CB200_ROUTE(true, true);
    else CB200_ROUTE(false, true);
    return launch_status();
  }
  if (experts <= 32 * kHeld) CB200_ROUTE(true, false);
  else CB200_ROUTE(false, false);
#undef CB200_ROUTE
  place_kernel<<<rows, kRouteThreads, smem, st>>>(rows, experts, top, counters, cu, token_of, place_of, chosen, static_cast<const uint4*>(x),
                                                  static_cast<uint4*>(placed), row_bytes / 16);
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
