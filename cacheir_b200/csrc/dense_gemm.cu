// Plain entry points of the dense tensor-core GEMM (dense_gemm.cuh).
#include "dense_gemm.cuh"

namespace cb200 {
namespace {

struct Shape { int mt, split; };
Shape choose_shape(int T, int N, int K, int batch) {
  const int n_tiles = (N + kTileN - 1) / kTileN * batch;
  int mt = T <= 16 ? 16 : T <= 32 ? 32 : T <= 64 ? 64 : 128;
  if (T >= 256 && n_tiles * ((T + 255) / 256) >= kNumSMs) mt = 256;
  const int tiles = n_tiles * ((T + mt - 1) / mt);
  const int kblocks = (K + kBlockK - 1) / kBlockK;
  const int slots = kNumSMs * ctas_per_sm(mt);
  int split = 1;
  while (split < 8 && tiles * split * 2 <= slots && kblocks / (split * 2) >= 4) split *= 2;
  return {mt, split};
}

template <int EPI>
int launch_mt(const cacheir_b200_dense_args& p, cudaStream_t stream) {
  const Shape s = choose_shape(p.T, p.N, p.K, p.batch);
  switch (s.mt) {
    case 16: return launch<EPI, 16, false>(p, s.split, stream, {});
    case 32: return launch<EPI, 32, false>(p, s.split, stream, {});
    case 64: return launch<EPI, 64, false>(p, s.split, stream, {});
    case 128: return launch<EPI, 128, false>(p, s.split, stream, {});
    default: return launch<EPI, 256, false>(p, s.split, stream, {});
  }
}

}  // namespace

}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_dense_supported(int K, long long w_stride, long long x_stride, int batch, int x_batch_cols) {
  return K > 0 && w_stride % 8 == 0 && x_stride % 8 == 0 && (batch <= 1 || x_batch_cols % 8 == 0) ? 1 : 0;
}

extern "C" int cacheir_b200_dense_gemm(const cacheir_b200_dense_args* args, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  cacheir_b200_dense_args p = *args;
  if (p.T <= 0 || p.N <= 0) return 0;
  if (p.batch < 1) p.batch = 1;
  if (p.K <= 0 || !p.x || !p.w) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_dense_supported(p.K, p.w_stride, p.x_stride, p.batch, p.x_batch_cols) || !aligned_to(p.x, 16) || !aligned_to(p.w, 16))
    return CACHEIR_B200_EALIGN;
  if (p.w_stride < p.K || p.x_stride < static_cast<long long>(p.x_batch_cols) * (p.batch - 1) + p.K) return CACHEIR_B200_EINVAL;
  if (p.batch > 1 && (p.w_batch_rows < p.N || p.bias)) return CACHEIR_B200_EINVAL;
  if ((static_cast<long long>(p.N) + kTileN - 1) / kTileN * p.batch > 65535) return CACHEIR_B200_ELIMIT;
  const bool tail_ok = p.tail_cols >= 0 && p.tail_cols <= p.N && (p.tail_cols == 0 || (p.tail && p.batch == 1));
  cudaStream_t st = as_stream(stream);
  switch (p.epilogue) {
    case CACHEIR_B200_DENSE_BF16: return p.y && tail_ok ? launch_mt<CACHEIR_B200_DENSE_BF16>(p, st) : CACHEIR_B200_EINVAL;
    case CACHEIR_B200_DENSE_F32: return p.y ? launch_mt<CACHEIR_B200_DENSE_F32>(p, st) : CACHEIR_B200_EINVAL;
    case CACHEIR_B200_DENSE_SILU: return p.y && tail_ok ? launch_mt<CACHEIR_B200_DENSE_SILU>(p, st) : CACHEIR_B200_EINVAL;
    case CACHEIR_B200_DENSE_RELU2: return p.y ? launch_mt<CACHEIR_B200_DENSE_RELU2>(p, st) : CACHEIR_B200_EINVAL;
    case CACHEIR_B200_DENSE_GEGLU:
    case CACHEIR_B200_DENSE_SWIGLU:
    case CACHEIR_B200_DENSE_CLAMPED_GLU:
      if (!p.y || !tail_ok || (p.N - p.tail_cols) % 2 != 0 || p.batch != 1)
        return CACHEIR_B200_EINVAL;
      if (p.epilogue == CACHEIR_B200_DENSE_GEGLU) return launch_mt<CACHEIR_B200_DENSE_GEGLU>(p, st);
      if (p.epilogue == CACHEIR_B200_DENSE_SWIGLU) return launch_mt<CACHEIR_B200_DENSE_SWIGLU>(p, st);
      return launch_mt<CACHEIR_B200_DENSE_CLAMPED_GLU>(p, st);
    case CACHEIR_B200_DENSE_GATED:
      return p.y && p.gate ? launch_mt<CACHEIR_B200_DENSE_GATED>(p, st) : CACHEIR_B200_EINVAL;
    case CACHEIR_B200_DENSE_GELU_EMBED:
      if (!p.y || !p.ids || !p.table || p.vocab <= 0 || p.batch != 1) return CACHEIR_B200_EINVAL;
      return launch_mt<CACHEIR_B200_DENSE_GELU_EMBED>(p, st);
    case CACHEIR_B200_DENSE_RESIDUAL:
      if (!p.residual || !p.norm_w || !p.norm_b || p.batch != 1) return CACHEIR_B200_EINVAL;
      if (p.next_mode != CACHEIR_B200_NEXT_NONE && !p.next_out) return CACHEIR_B200_EINVAL;
      if (p.next_mode == CACHEIR_B200_NEXT_DYT && (!p.next_w || !p.next_b)) return CACHEIR_B200_EINVAL;
      return launch_mt<CACHEIR_B200_DENSE_RESIDUAL>(p, st);
    default: return CACHEIR_B200_EINVAL;
  }
}

extern "C" int cacheir_b200_ragged_device_status(int reset) { return device_status_word(g_dense_status, reset != 0); }
