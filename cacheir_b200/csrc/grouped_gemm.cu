// One GEMM per expert over the places of a routed step: the grouped form of dense_gemm.cuh, and its float32 counterpart.
#include "cacheir_b200_experts.h"
#include "dense_gemm.cuh"

namespace cb200 {
namespace {

constexpr int kAllRows = 64;      // a step of at most this many rows is multiplied as a whole by every expert in use

// Tile width from the mean number of places per expert: a wider tile reads an expert's weights fewer times, a narrower one
// leaves less of its last tile unused.
int choose_tile(int places, int experts, const Groups& g) {
  if (g.place_of) return g.x_rows <= 16 ? 16 : g.x_rows <= 32 ? 32 : 64;
  const int mean = (places + experts - 1) / experts;
  return mean <= 8 ? 16 : mean <= 16 ? 32 : mean <= 48 ? 64 : mean <= 1024 ? 128 : 256;
}

int choose_split(int places, int experts, int N, int K, int mt, const Groups& g) {
  const int items = (g.place_of ? 0 : places / mt) + (places < experts ? places : experts);
  const int tiles = (N + kTileN - 1) / kTileN * items;
  const int kblocks = (K + kBlockK - 1) / kBlockK;
  int split = 1;
  while (split < 8 && tiles * split * 2 <= kNumSMs * ctas_per_sm(mt) && kblocks / (split * 2) >= 4) split *= 2;
  return split;
}

template <int EPI>
int launch_grouped(const cacheir_b200_dense_args& p, const Groups& g, cudaStream_t st) {
  const int mt = choose_tile(p.T, p.batch, g);
  const int split = choose_split(p.T, p.batch, p.N, p.K, mt, g);
  switch (mt) {
    case 16: return launch<EPI, 16, true>(p, split, st, g);
    case 32: return launch<EPI, 32, true>(p, split, st, g);
    case 64: return launch<EPI, 64, true>(p, split, st, g);
    case 128: return launch<EPI, 128, true>(p, split, st, g);
    default: return launch<EPI, 256, true>(p, split, st, g);
  }
}

// ---- float32 arithmetic, any extents: 16 places x 64 columns per CTA -----------------------------------------------
constexpr int kSimpleRows = 16, kSimpleCols = 64, kSimpleK = 16;
template <typename T>
__global__ void __launch_bounds__(256)
grouped_simple_kernel(const T* __restrict__ x, const T* __restrict__ w, T* __restrict__ y, const int32_t* __restrict__ cu,
                      const int32_t* __restrict__ token_of, int experts, int N, int K, long long ws, long long xs, long long ys) {
  __shared__ float sx[kSimpleK][kSimpleRows + 1], sw[kSimpleK][kSimpleCols + 4];
  const RaggedItem it = find_item(cu, experts, kSimpleRows, blockIdx.x);
  if (it.seg < 0) return;
  w += static_cast<long long>(it.seg) * N * ws;
  const int n0 = blockIdx.y * kSimpleCols, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int place = it.row0 + min(ty, it.count - 1);
  const long long src = token_of ? token_of[place] : place;
  float acc[4] = {};
  for (int k0 = 0; k0 < K; k0 += kSimpleK) {
    sx[tx][ty] = k0 + tx < K ? Elem<T>::ld(x + src * xs + k0 + tx) : 0.f;
    for (int i = threadIdx.x; i < kSimpleCols * kSimpleK; i += 256) {
      const int r = i / kSimpleK, k = i % kSimpleK;
      sw[k][r] = (n0 + r < N && k0 + k < K) ? Elem<T>::ld(w + static_cast<long long>(n0 + r) * ws + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSimpleK; ++k) {
      const float a = sx[k][ty];
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[j] = fmaf(a, sw[k][tx * 4 + j], acc[j]);
    }
    __syncthreads();
  }
  if (ty < it.count)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (n0 + tx * 4 + j < N) Elem<T>::st(y + static_cast<long long>(place) * ys + n0 + tx * 4 + j, acc[j]);
}

}  // namespace

int tied_attention_status(bool reset);
int tied_prompt_status(bool reset);

}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_grouped_all_rows(void) { return kAllRows; }

extern "C" int cacheir_b200_grouped_gemm(const cacheir_b200_dense_args* args, const int32_t* cu, const int32_t* place_of, int top, int x_rows,
                                         void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_dense_args& p = *args;
  if (p.T <= 0 || p.N <= 0) return 0;
  if (p.batch < 1 || p.K <= 0 || !p.x || !p.w || !p.y || !cu || x_rows <= 0 || p.bias || p.tail_cols != 0 || p.w_batch_rows < p.N ||
      (place_of && top < 1))
    return CACHEIR_B200_EINVAL;
  if (place_of && x_rows > kAllRows) return CACHEIR_B200_ELIMIT;
  if (p.w_stride % 8 != 0 || p.x_stride % 8 != 0 || !aligned_to(p.x, 16) || !aligned_to(p.w, 16)) return CACHEIR_B200_EALIGN;
  if (p.w_stride < p.K || p.x_stride < p.K) return CACHEIR_B200_EINVAL;
  const Groups g{cu, place_of, top, x_rows};
  cudaStream_t st = as_stream(stream);
  switch (p.epilogue) {
    case CACHEIR_B200_DENSE_BF16: return launch_grouped<CACHEIR_B200_DENSE_BF16>(p, g, st);
    case CACHEIR_B200_DENSE_SWIGLU: return p.N % 2 ? CACHEIR_B200_EINVAL : launch_grouped<CACHEIR_B200_DENSE_SWIGLU>(p, g, st);
    case CACHEIR_B200_DENSE_CLAMPED_GLU: return p.N % 2 ? CACHEIR_B200_EINVAL : launch_grouped<CACHEIR_B200_DENSE_CLAMPED_GLU>(p, g, st);
    default: return CACHEIR_B200_EINVAL;
  }
}

extern "C" int cacheir_b200_grouped_simple(const void* x, const void* w, void* y, const int32_t* cu, const int32_t* token_of, int places,
                                           int experts, int N, int K, long long w_stride, long long x_stride, long long y_stride,
                                           int dtype, void* stream) {
  if (places <= 0 || N <= 0) return 0;
  if (!x || !w || !y || !cu || experts < 1 || K <= 0) return CACHEIR_B200_EINVAL;
  const dim3 grid(ragged_items(places, experts, kSimpleRows), (N + kSimpleCols - 1) / kSimpleCols);
  if (grid.y > 65535) return CACHEIR_B200_ELIMIT;
  CB200_HYBRID_DTYPE(dtype, (grouped_simple_kernel<T><<<grid, 256, 0, as_stream(stream)>>>(
                                static_cast<const T*>(x), static_cast<const T*>(w), static_cast<T*>(y), cu, token_of, experts, N, K,
                                w_stride, x_stride, y_stride)));
  return launch_status();
}

extern "C" int cacheir_b200_experts_device_status(int reset) {
  const int gemm = device_status_word(g_dense_status, reset != 0), step = tied_attention_status(reset != 0), prompt = tied_prompt_status(reset != 0);
  return gemm != 0 ? gemm : step != 0 ? step : prompt;
}
