// Around the experts' products: which tokens go to which expert, and the weighted sum of what comes back with the
// residual add and the norm before or behind it.
#include "cacheir_b200_experts.h"
#include "residual_rows.cuh"

namespace cb200 {
namespace {

constexpr int kRouteThreads = 256;      // a warp per token
constexpr int kHeld = 4;                // logits a lane keeps in registers

// Softmax scores plus correction of one token's logits into `choice` [scored], -inf outside the rule's best groups; `best` has
// room for a score per group. Returns (maximum, 1 / sum) of the softmax. One warp.
__device__ __forceinline__ float2 softmax_choices(const float* z, int scored, const cacheir_b200_route_rule& rule, float* choice, float* best) {
  const int lane = threadIdx.x & 31;
  float m = -INFINITY, sum = 0.f;
  for (int e = lane; e < scored; e += 32) m = fmaxf(m, z[e]);
  m = warp_max(m);
  for (int e = lane; e < scored; e += 32) {
    const float p = expf(z[e] - m);
    choice[e] = p;
    sum += p;
  }
  const float inv = 1.f / warp_sum(sum);
  for (int e = lane; e < scored; e += 32) choice[e] = choice[e] * inv + (rule.correction ? rule.correction[e] : 0.f);
  __syncwarp();
  if (rule.keep < rule.groups) {
    const int size = scored / rule.groups;
    for (int g = lane; g < rule.groups; g += 32) {
      float b = -INFINITY;
      for (int e = g * size; e < (g + 1) * size; ++e) b = fmaxf(b, choice[e]);
      best[g] = b;
    }
    __syncwarp();
    for (int g = lane; g < rule.groups; g += 32) {
      int ahead = 0;
      for (int o = 0; o < rule.groups; ++o) ahead += best[o] > best[g] || (best[o] == best[g] && o < g);
      if (ahead >= rule.keep)
        for (int e = g * size; e < (g + 1) * size; ++e) choice[e] = -INFINITY;
    }
    __syncwarp();
  }
  return make_float2(m, inv);
}

// The warp's token: its choices in order, each with its rank among the tokens of that expert (in no particular order).
// Choices go by z, or (SOFTMAX) by the scores in `choice`. Index experts and up: the token itself, which needs no place.
template <bool HELD, bool SOFTMAX>
__device__ __forceinline__ void choose(const float* logits, bool real, int row, int experts, int scored, int top, const cacheir_b200_route_rule& rule,
                                       float* choice, int32_t* counters, int32_t* place_of, float* weight, int32_t* chosen) {
  const int lane = threadIdx.x & 31;
  float2 sm = make_float2(0.f, 0.f);
  if (SOFTMAX) sm = softmax_choices(logits, scored, rule, choice, choice + scored);
  const float* z = SOFTMAX ? choice : logits;
  float held[kHeld];
  if (HELD) {
#pragma unroll
    for (int i = 0; i < kHeld; ++i) held[i] = lane + 32 * i < scored ? z[lane + 32 * i] : 0.f;
  }
  float bound = INFINITY;               // the last choice: what follows it in (value descending, index ascending) order is next
  int after = -1, mine = -1;
  float mine_z = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = scored;
    auto look = [&](int e, float v) {
      if ((v < bound || (v == bound && e > after)) && (v > best || at == scored)) { best = v; at = e; }
    };
    if (HELD) {
#pragma unroll
      for (int i = 0; i < kHeld; ++i)
        if (lane + 32 * i < scored) look(lane + 32 * i, held[i]);
    } else {
      for (int e = lane; e < scored; e += 32) look(e, z[e]);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
      const float v = __shfl_xor_sync(0xffffffffu, best, off);
      const int e = __shfl_xor_sync(0xffffffffu, at, off);
      if (e < scored && (at == scored || v > best || (v == best && e < at))) { best = v; at = e; }
    }
    bound = best;
    after = at;
    if (lane == k % 32) { mine = at; mine_z = best; }
    if (k % 32 == 31 || k == top - 1) { // the lanes record what they hold: one round of atomics for up to 32 choices
      const int j = k / 32 * 32 + lane;
      if (j <= k) {
        const bool take = real && mine < scored;       // (a row of NaNs chooses nothing)
        const float score = !take ? 0.f : SOFTMAX ? expf(logits[mine] - sm.x) * sm.y : sigmoid_exact(mine_z);
        chosen[row * top + j] = take ? mine : -1;
        weight[row * top + j] = score * rule.scale;
        place_of[row * top + j] = !take ? CACHEIR_B200_PLACE_NONE : mine < experts ? atomicAdd(&counters[mine], 1) : CACHEIR_B200_PLACE_SELF;
      }
    }
  }
}

// Every block chooses for its tokens and counts; the block that finishes last turns counts into places (nobody waits).
// PLACE false: choices and ranks only.
template <bool HELD, bool PLACE, bool SOFTMAX>
__global__ void __launch_bounds__(kRouteThreads)
route_kernel(const float* __restrict__ logits, long long stride, const int32_t* __restrict__ row_seg, int rows, int experts, int top,
             const cacheir_b200_route_rule rule, int32_t* counters, int32_t* __restrict__ cu, int32_t* __restrict__ token_of, int32_t* place_of,
             float* __restrict__ weight, int32_t* chosen) {
  extern __shared__ int s_first[];      // [experts + 1] (SOFTMAX: then a warp's choice scores, and its groups' best)
  __shared__ int s_sum[kRouteThreads / 32];
  __shared__ bool s_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = blockIdx.x * (kRouteThreads / 32) + warp;
  const int scored = experts + rule.identity;
  float* choice = reinterpret_cast<float*>(s_first + experts + 1) + warp * (scored + rule.groups);
  if (row < rows)
    choose<HELD, SOFTMAX>(logits + static_cast<long long>(row) * stride, row_seg[row] >= 0, row, experts, scored, top, rule, choice, counters, place_of,
                          weight, chosen);
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
    if (e < 0 || rank < 0) continue;
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
    const int e = chosen[row * top + k], rank = place_of[row * top + k];
    int before = 0;
    for (int i = lane; i < e && rank >= 0; i += 32) before += s_count[i];
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) before += __shfl_xor_sync(0xffffffffu, before, off);
    if (lane == 0) {
      const int place = rank < 0 ? rank : before + rank;
      s_place[k] = place;
      if (rank >= 0) {
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

// residual += sum of the chosen experts' rows by weight + shared row * sigmoid(its gate). `self` and `nx.out` may be one buffer.
template <typename T, int VEC>
__global__ void __launch_bounds__(512)
combine_add_kernel(float* x, const T* __restrict__ y, const int32_t* __restrict__ place_of, const float* __restrict__ weight, int top,
                   const T* self, const T* __restrict__ shared, const float* __restrict__ shared_gate, long long shared_gate_stride, int width,
                   RowNext nx) {
  __shared__ float scratch[32];
  const size_t row = blockIdx.x;
  float own = 0.f;                      // weight of the token itself
  for (int k = 0; k < top; ++k)
    if (place_of[row * top + k] == CACHEIR_B200_PLACE_SELF) own += weight[row * top + k];
  const float by = shared_gate ? sigmoid_exact(shared_gate[row * shared_gate_stride]) : 1.f;
  finish_row<T, VEC>(x + row * width, row, width, nx, scratch, [&](int c, float (&s)[VEC]) {
    float m[VEC] = {}, v[VEC];
    if (shared) {
      load_vec<T, VEC>(shared + row * width + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) m[i] = v[i] * by;
    }
    if (own != 0.f) {
      load_vec<T, VEC>(self + row * width + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) m[i] = fmaf(own, v[i], m[i]);
    }
    for (int k = 0; k < top; ++k) {
      const int place = place_of[row * top + k];
      if (place < 0) continue;
      const float a = weight[row * top + k];
      load_vec<T, VEC>(y + static_cast<size_t>(place) * width + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) m[i] = fmaf(a, v[i], m[i]);
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) s[i] += m[i];
  });
}

}  // namespace
}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_route(const float* logits, long long stride, const int32_t* row_seg, int rows, int experts, int top,
                                  const cacheir_b200_route_rule* rule, int32_t* counters, int32_t* cu, int32_t* token_of, int32_t* place_of, float* weight, int32_t* chosen,
                                  const void* x, void* placed, int row_bytes, void* stream) {
  if (rows <= 0) return 0;
  if (!rule || rule->identity < 0 || experts < 1) return CACHEIR_B200_EINVAL;
  const int scored = experts + rule->identity;
  if (!rule->softmax && (rule->correction || rule->groups > 1)) return CACHEIR_B200_EINVAL;
  if (rule->softmax && (rule->groups < 1 || rule->keep < 1 || rule->keep > rule->groups || scored % rule->groups != 0 ||
                        top > scored / rule->groups * rule->keep))
    return CACHEIR_B200_EINVAL;
  if (!logits || !row_seg || top < 1 || top > scored || stride < scored || !counters || !cu || !token_of || !place_of ||
      !weight || !chosen || (placed && (!x || row_bytes <= 0)))
    return CACHEIR_B200_EINVAL;
  if (placed && (row_bytes % 16 != 0 || !aligned_to(x, 16) || !aligned_to(placed, 16))) return CACHEIR_B200_EALIGN;
  const size_t smem = static_cast<size_t>(experts + top + 1) * 4;
  const size_t choices = rule->softmax ? static_cast<size_t>(kRouteThreads / 32) * (scored + rule->groups) * 4 : 0;
  const size_t first = static_cast<size_t>(experts + 1) * 4;
  if (smem > 40 * 1024 || first + choices > 40 * 1024) return CACHEIR_B200_ELIMIT;
  const int blocks = (rows + 7) / 8;
  cudaStream_t st = as_stream(stream);
  const bool held = scored <= 32 * kHeld;
#define CB200_ROUTE(HELD, PLACE, SOFTMAX)                                                                                              \
  route_kernel<HELD, PLACE, SOFTMAX><<<blocks, kRouteThreads, PLACE || SOFTMAX ? first + choices : 0, st>>>(                            \
      logits, stride, row_seg, rows, experts, top, *rule, counters, cu, token_of, place_of, weight, chosen)
#define CB200_ROUTE_RULE(PLACE)                          \
  if (rule->softmax && held) CB200_ROUTE(true, PLACE, true);      \
  else if (rule->softmax) CB200_ROUTE(false, PLACE, true);        \
  else if (held) CB200_ROUTE(true, PLACE, false);                 \
  else CB200_ROUTE(false, PLACE, false)
  if (!placed) {
    CB200_ROUTE_RULE(true);
    return launch_status();
  }
  CB200_ROUTE_RULE(false);
#undef CB200_ROUTE_RULE
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

extern "C" int cacheir_b200_combine_residual(float* residual, const void* y, const int32_t* place_of, const float* weight, int top, const void* self,
                                             const void* shared, const float* shared_gate, long long shared_gate_stride, int rows, int width,
                                             int next_mode, const float* next_w, const float* next_b, float next_alpha, void* next_out, int dtype,
                                             void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !y || !place_of || !weight || top < 1 || !self || next_b || !row_next_ok(next_mode, next_w, next_out)) return CACHEIR_B200_EINVAL;
  const RowNext nx{next_mode, next_w, next_alpha, next_out};
  const bool vec = width % 4 == 0 && aligned_to(residual, 16) && aligned_to(y, 16) && aligned_to(self, 16) && aligned_to(shared, 16) &&
                   row_next_aligned(next_mode, next_w, next_out);
#define CB200_COMBINE(VEC)                                                                                                                 \
  combine_add_kernel<T, VEC><<<rows, 512, 0, as_stream(stream)>>>(residual, static_cast<const T*>(y), place_of, weight, top,                \
                                                                 static_cast<const T*>(self), static_cast<const T*>(shared), shared_gate, \
                                                                 shared_gate_stride, width, nx)
  CB200_HYBRID_DTYPE(dtype, {
    if (vec) CB200_COMBINE(4);
    else CB200_COMBINE(1);
  });
#undef CB200_COMBINE
  return launch_status();
}
