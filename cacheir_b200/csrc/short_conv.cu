// Short causal convolution per channel with silu over the rows of a ragged step, sm_100a. A thread owns VEC neighbouring channels of
// a piece of a sequence's rows and slides a window of the last inputs along it. The piece with a sequence's first row reads the
// inputs that earlier steps left in the slot and, since the last rows' inputs are in memory anyway, also writes the new ones:
// nobody else touches the slot.
#include "cacheir_b200_delta.h"
#include "hybrid_common.cuh"
#include "ragged.cuh"

namespace cb200 {
namespace {

using Args = cacheir_b200_conv_args;
constexpr int kPieceRows = 32;         // at least taps - 1, so that only the first piece needs the slot
constexpr int kMaxTaps = kPieceRows;
constexpr int kThreads = 128;

__device__ __forceinline__ float* slot_inputs(const Args& a, int seg) {
  return a.state + static_cast<size_t>(min(max(a.slots[seg], 0), a.num_slots - 1)) * a.slot_stride;
}

// TAPS > 0: window and weights in registers
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kThreads)
short_conv_kernel(const Args a) {
  constexpr int H = TAPS - 1, U = 8;   // inputs kept; rows requested at a time
  const RaggedItem it = find_item(a.cu_rows, a.segments, kPieceRows, blockIdx.x);
  const int c = (blockIdx.y * kThreads + threadIdx.x) * VEC;
  if (it.seg < 0 || c >= a.channels) return;
  const bool first = static_cast<int>(blockIdx.x) == it.first;
  const T* x = static_cast<const T*>(a.x) + static_cast<size_t>(it.row0) * a.stride + c;
  T* out = static_cast<T*>(a.out) + static_cast<size_t>(it.row0) * a.out_stride + c;
  float* kept = H > 0 ? slot_inputs(a, it.seg) + c : nullptr;
  float w[VEC][TAPS], b[VEC], past[H > 0 ? H : 1][VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    b[i] = a.bias ? a.bias[c + i] : 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[i][j] = a.w[static_cast<size_t>(c + i) * TAPS + j];
  }
  const bool fresh = first && a.positions[it.row0] == 0;
#pragma unroll
  for (int j = 0; j < H; ++j) {
    if (!first) {
      load_vec<T, VEC>(x + static_cast<long long>(j - H) * a.stride, past[j]);
    } else if (!fresh) {
      load_vec<float, VEC>(kept + static_cast<size_t>(j) * a.channels, past[j]);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) past[j][i] = 0.f;
    }
  }
  if (H > 0 && first) {                // the inputs the next step will need
    const int rows = a.cu_rows[it.seg + 1] - it.row0;
#pragma unroll
    for (int j = 0; j < H; ++j) {
      const int t = rows - H + j;      // row of the segment, negative: an old input
      float v[VEC];
      if (t >= 0) {
        load_vec<T, VEC>(x + static_cast<long long>(t) * a.stride, v);
      } else {
#pragma unroll
        for (int k = 0; k < H; ++k)
          if (k == t + H)
#pragma unroll
            for (int i = 0; i < VEC; ++i) v[i] = past[k][i];
      }
      store_vec<float, VEC>(kept + static_cast<size_t>(j) * a.channels, v);
    }
  }
  for (int r0 = 0; r0 < it.count; r0 += U) {
    float v[U][VEC];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (r0 + u < it.count) load_vec<T, VEC>(x + static_cast<long long>(r0 + u) * a.stride, v[u]);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (r0 + u >= it.count) break;
      float y[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        y[i] = b[i];
#pragma unroll
        for (int j = 0; j < H; ++j) y[i] = fmaf(w[i][j], past[j][i], y[i]);
        y[i] = silu_exact(fmaf(w[i][TAPS - 1], v[u][i], y[i]));
#pragma unroll
        for (int j = 0; j + 1 < H; ++j) past[j][i] = past[j + 1][i];
        if (H > 0) past[H > 0 ? H - 1 : 0][i] = v[u][i];
      }
      store_vec<T, VEC>(out + static_cast<long long>(r0 + u) * a.out_stride, y);
    }
  }
}

// any number of taps up to kMaxTaps
template <typename T>
__global__ void __launch_bounds__(kThreads)
long_conv_kernel(const Args a) {
  const RaggedItem it = find_item(a.cu_rows, a.segments, kPieceRows, blockIdx.x);
  const int c = blockIdx.y * kThreads + threadIdx.x, H = a.taps - 1;
  if (it.seg < 0 || c >= a.channels) return;
  const bool first = static_cast<int>(blockIdx.x) == it.first, fresh = first && a.positions[it.row0] == 0;
  const T* x = static_cast<const T*>(a.x) + static_cast<size_t>(it.row0) * a.stride + c;
  float* kept = slot_inputs(a, it.seg) + c;
  auto input = [&](int t) {            // row t of this piece, negative: before it
    if (t >= 0 || !first) return Elem<T>::ld(x + static_cast<long long>(t) * a.stride);
    return fresh ? 0.f : kept[static_cast<size_t>(t + H) * a.channels];
  };
  for (int r = 0; r < it.count; ++r) {
    float y = a.bias ? a.bias[c] : 0.f;
    for (int j = 0; j <= H; ++j) y = fmaf(a.w[static_cast<size_t>(c) * a.taps + j], input(r - H + j), y);
    Elem<T>::st(static_cast<T*>(a.out) + static_cast<size_t>(it.row0 + r) * a.out_stride + c, silu_exact(y));
  }
  if (first) {
    const int rows = a.cu_rows[it.seg + 1] - it.row0;
    for (int j = 0; j < H; ++j) kept[static_cast<size_t>(j) * a.channels] = input(rows - H + j);      // (reads at or behind what it writes)
  }
}

template <typename T, int VEC>
int launch_conv(const Args& a, cudaStream_t st) {
  const int items = ragged_items(a.rows, a.segments, kPieceRows), per_block = kThreads * VEC;
  const dim3 grid(items, (a.channels + per_block - 1) / per_block);
  switch (a.taps) {
    case 1: short_conv_kernel<T, VEC, 1><<<grid, kThreads, 0, st>>>(a); break;
    case 2: short_conv_kernel<T, VEC, 2><<<grid, kThreads, 0, st>>>(a); break;
    case 3: short_conv_kernel<T, VEC, 3><<<grid, kThreads, 0, st>>>(a); break;
    case 4: short_conv_kernel<T, VEC, 4><<<grid, kThreads, 0, st>>>(a); break;
    default: long_conv_kernel<T><<<dim3(items, (a.channels + kThreads - 1) / kThreads), kThreads, 0, st>>>(a);
  }
  return launch_status();
}

}  // namespace
}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_short_conv(const cacheir_b200_conv_args* args, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_conv_args& a = *args;
  if (a.rows <= 0 || a.channels <= 0) return 0;
  if (!a.positions || !a.cu_rows || !a.slots || !a.x || !a.w || !a.state || !a.out || a.segments <= 0 || a.taps <= 0 || a.num_slots <= 0 ||
      a.stride < a.channels || a.out_stride < a.channels || a.slot_stride < static_cast<long long>(a.taps - 1) * a.channels)
    return CACHEIR_B200_EINVAL;
  if (a.taps > kMaxTaps) return CACHEIR_B200_ELIMIT;
  const int quad = 4 * (a.dtype == CACHEIR_B200_F32 ? 4 : 2);
  const bool vec = a.channels % 4 == 0 && a.stride % 4 == 0 && a.out_stride % 4 == 0 && a.slot_stride % 4 == 0 && aligned_to(a.x, quad) &&
                   aligned_to(a.out, quad) && aligned_to(a.state, 16);
  CB200_HYBRID_DTYPE(a.dtype, return vec ? launch_conv<T, 4>(a, as_stream(stream)) : launch_conv<T, 1>(a, as_stream(stream)));
  return CACHEIR_B200_EUNSUPPORTED;
}
