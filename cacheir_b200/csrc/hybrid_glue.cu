// Row operators of the hybrid families that are not a GEMM epilogue: embedding into the 32-bit residual stream, Dynamic
// Tanh, the (RMS-normed, scaled) residual add, layer norms, the gated RMS norms behind a recurrence, and the stand-alone forms of the dense
// kernel's epilogues (used in 32-bit runs and for extents the tensor-core kernel does not take).
#include "residual_rows.cuh"

namespace cb200 {
namespace {

struct NextArgs {
  int mode;
  const float* w;
  const float* b;
  float alpha;
  void* out;
};

template <typename T>
__device__ __forceinline__ void leave_next(const NextArgs& nx, size_t idx, int c, float s) {
  if (nx.mode == CACHEIR_B200_NEXT_DYT) Elem<T>::st(static_cast<T*>(nx.out) + idx, fmaf(tanhf(nx.alpha * s), nx.w[c], nx.b[c]));
  else if (nx.mode == CACHEIR_B200_NEXT_COPY) Elem<T>::st(static_cast<T*>(nx.out) + idx, s);
}

template <typename T>
__global__ void __launch_bounds__(256)
scaled_embedding_kernel(const T* __restrict__ table, const int64_t* __restrict__ ids, float* __restrict__ x, int width, int vocab,
                        float scale, NextArgs nx) {
  const size_t row = blockIdx.x;
  const int64_t id = min(max(ids[row], static_cast<int64_t>(0)), static_cast<int64_t>(vocab - 1));
  for (int c = blockIdx.y * 256 + threadIdx.x; c < width; c += gridDim.y * 256) {
    const float s = Elem<T>::ld(table + id * width + c) * scale;
    x[row * width + c] = s;
    leave_next<T>(nx, row * width + c, c, s);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
dyt_rows_kernel(const float* __restrict__ x, const int32_t* __restrict__ row_index, const float* __restrict__ w,
                const float* __restrict__ b, float alpha, T* __restrict__ out, int width) {
  const size_t row = blockIdx.x;
  const size_t src = row_index ? static_cast<size_t>(max(row_index[row], 0)) : row;
  for (int c = blockIdx.y * 256 + threadIdx.x; c < width; c += gridDim.y * 256)
    Elem<T>::st(out + row * width + c, fmaf(tanhf(alpha * x[src * width + c]), w[c], b[c]));
}

template <typename T, int VEC>
__global__ void __launch_bounds__(512)
rms_rows_kernel(const float* __restrict__ x, const int32_t* __restrict__ row_index, const float* __restrict__ w, float eps,
                T* __restrict__ out, int width) {
  __shared__ float scratch[32];
  const size_t row = blockIdx.x;
  const float* xr = x + (row_index ? static_cast<size_t>(max(row_index[row], 0)) : row) * width;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < width; c += 512 * VEC) {
    float v[VEC];
    load_vec<float, VEC>(xr + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, scratch) / static_cast<float>(width) + eps);
  for (int c = threadIdx.x * VEC; c < width; c += 512 * VEC) {
    float v[VEC], wv[VEC];
    load_vec<float, VEC>(xr + c, v);
    load_vec<float, VEC>(w + c, wv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * inv * wv[i];
    store_vec<T, VEC>(out + row * width + c, v);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
residual_dyt_kernel(float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ w, const float* __restrict__ b,
                    float alpha, int width, NextArgs nx) {
  const size_t row = blockIdx.x;
  for (int c = blockIdx.y * 256 + threadIdx.x; c < width; c += gridDim.y * 256) {
    const size_t i = row * width + c;
    const float s = x[i] + fmaf(tanhf(alpha * Elem<T>::ld(y + i)), w[c], b[c]);
    x[i] = s;
    leave_next<T>(nx, i, c, s);
  }
}

constexpr int kRowThreads = 512;

template <typename T, int VEC>
__global__ void __launch_bounds__(kRowThreads)
residual_rms_kernel(float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ w, float eps, int width, NextArgs nx) {
  __shared__ float scratch[32];
  const size_t row = blockIdx.x;
  const T* yr = y + row * width;
  float* xr = x + row * width;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < width; c += kRowThreads * VEC) {
    float v[VEC];
    load_vec<T, VEC>(yr + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, scratch) / static_cast<float>(width) + eps);
  for (int c = threadIdx.x * VEC; c < width; c += kRowThreads * VEC) {
    float v[VEC], wv[VEC], s[VEC];
    load_vec<T, VEC>(yr + c, v);
    load_vec<float, VEC>(w + c, wv);
    load_vec<float, VEC>(xr + c, s);
#pragma unroll
    for (int i = 0; i < VEC; ++i) s[i] = fmaf(v[i] * inv, wv[i], s[i]);
    store_vec<float, VEC>(xr + c, s);
    if (nx.mode == CACHEIR_B200_NEXT_DYT) {
      float nw[VEC], nb[VEC];
      load_vec<float, VEC>(nx.w + c, nw);
      load_vec<float, VEC>(nx.b + c, nb);
#pragma unroll
      for (int i = 0; i < VEC; ++i) s[i] = fmaf(tanhf(nx.alpha * s[i]), nw[i], nb[i]);
    }
    if (nx.mode != CACHEIR_B200_NEXT_NONE) store_vec<T, VEC>(static_cast<T*>(nx.out) + row * width + c, s);
  }
}

// residual = table[ids] * scale, or that much more
template <typename T, int VEC, bool ADD>
__global__ void __launch_bounds__(kRowThreads)
embedding_rows_kernel(const T* __restrict__ table, const int64_t* __restrict__ ids, float* x, int width, int vocab, float scale, RowNext nx) {
  __shared__ float scratch[32];
  const size_t row = blockIdx.x;
  const T* src = table + min(max(ids[row], static_cast<int64_t>(0)), static_cast<int64_t>(vocab - 1)) * width;
  finish_row<T, VEC>(x + row * width, row, width, nx, scratch, [&](int c, float (&s)[VEC]) {
    float v[VEC];
    load_vec<T, VEC>(src + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) s[i] = ADD ? s[i] + v[i] * scale : v[i] * scale;
  });
}

// HELD: a thread's columns stay in registers from the first read to the last write
constexpr int kAddThreads = 256, kAddPieces = 8;
template <typename T, int VEC, bool HELD>
__global__ void __launch_bounds__(kAddThreads)
residual_add_kernel(float* x, const T* __restrict__ y, const float* __restrict__ scale, int width, RowNext nx) {
  __shared__ float scratch[32];
  const size_t row = blockIdx.x;
  x += row * width;
  y += row * width;
  auto added = [&](int c, float (&s)[VEC]) {
    float v[VEC], f[VEC];
    load_vec<T, VEC>(y + c, v);
    if (scale) load_vec<float, VEC>(scale + c, f);
#pragma unroll
    for (int i = 0; i < VEC; ++i) s[i] = scale ? fmaf(v[i], f[i], s[i]) : s[i] + v[i];
  };
  if constexpr (HELD) {
    float s[kAddPieces][VEC], sum = 0.f;
    const bool centred = nx.mode == CACHEIR_B200_NEXT_LAYER;
    const auto column = [](int k) { return (k * kAddThreads + static_cast<int>(threadIdx.x)) * VEC; };
#pragma unroll
    for (int k = 0; k < kAddPieces; ++k)
      if (column(k) < width) load_vec<float, VEC>(x + column(k), s[k]);
#pragma unroll
    for (int k = 0; k < kAddPieces; ++k)
      if (column(k) < width) {
        added(column(k), s[k]);
#pragma unroll
        for (int i = 0; i < VEC; ++i) sum = centred ? sum + s[k][i] : fmaf(s[k][i], s[k][i], sum);
      }
    T* out = static_cast<T*>(nx.out) + row * width;
#pragma unroll
    for (int k = 0; k < kAddPieces; ++k)
      if (column(k) < width) {
        store_vec<float, VEC>(x + column(k), s[k]);
        if (nx.mode == CACHEIR_B200_NEXT_COPY) store_vec<T, VEC>(out + column(k), s[k]);
      }
    if (nx.mode != CACHEIR_B200_NEXT_RMS && !centred) return;
    float mean = 0.f;
    if (centred) {
      mean = block_sum_all(sum, scratch) / static_cast<float>(width);
      sum = 0.f;
#pragma unroll
      for (int k = 0; k < kAddPieces; ++k)
        if (column(k) < width)
#pragma unroll
          for (int i = 0; i < VEC; ++i) sum = fmaf(s[k][i] - mean, s[k][i] - mean, sum);
    }
    const float inv = 1.f / sqrtf(block_sum_all(sum, scratch) / static_cast<float>(width) + nx.eps);
#pragma unroll
    for (int k = 0; k < kAddPieces; ++k)
      if (column(k) < width) {
        float w[VEC];
        load_vec<float, VEC>(nx.w + column(k), w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) w[i] = (s[k][i] - mean) * inv * w[i];
        store_vec<T, VEC>(out + column(k), w);
      }
  } else {
    finish_row<T, VEC>(x, row, width, nx, scratch, added);
  }
}

// out[j] = layer norm of residual row row_index[j]
template <typename T, int VEC>
__global__ void __launch_bounds__(512)
layer_norm_rows_kernel(const float* __restrict__ x, const int32_t* __restrict__ row_index, const float* __restrict__ w, float eps,
                       T* __restrict__ out, int width) {
  __shared__ float scratch[32];
  const size_t row = blockIdx.x;
  const float* xr = x + (row_index ? static_cast<size_t>(max(row_index[row], 0)) : row) * width;
  float sum = 0.f, ss = 0.f;
  for (int c = threadIdx.x * VEC; c < width; c += 512 * VEC) {
    float v[VEC];
    load_vec<float, VEC>(xr + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) sum += v[i];
  }
  const float mean = block_sum_all(sum, scratch) / static_cast<float>(width);
  for (int c = threadIdx.x * VEC; c < width; c += 512 * VEC) {
    float v[VEC];
    load_vec<float, VEC>(xr + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i] - mean, v[i] - mean, ss);
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, scratch) / static_cast<float>(width) + eps);
  for (int c = threadIdx.x * VEC; c < width; c += 512 * VEC) {
    float v[VEC], wv[VEC];
    load_vec<float, VEC>(xr + c, v);
    load_vec<float, VEC>(w + c, wv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = (v[i] - mean) * inv * wv[i];
    store_vec<T, VEC>(out + row * width + c, v);
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
join_embedding_kernel(const float* __restrict__ x, const T* __restrict__ table, const int64_t* __restrict__ ids, T* __restrict__ out, int width,
                      int vocab) {
  const size_t row = blockIdx.x;
  const T* src = table + min(max(ids[row], static_cast<int64_t>(0)), static_cast<int64_t>(vocab - 1)) * width;
  for (int c = (blockIdx.y * 256 + threadIdx.x) * VEC; c < width; c += gridDim.y * 256 * VEC) {
    float v[VEC];
    load_vec<float, VEC>(x + row * width + c, v);
    store_vec<T, VEC>(out + row * 2 * width + c, v);
    load_vec<T, VEC>(src + c, v);
    store_vec<T, VEC>(out + row * 2 * width + width + c, v);
  }
}

// HELD: a thread's columns (PIECES vectors at most) stay in registers from the first read to the last write, and what a later
// step needs is requested before the sums.
constexpr int kPairThreads = 256, kPairPieces = 4;
template <typename T, int VEC, bool HELD>
__global__ void __launch_bounds__(kPairThreads)
residual_rms_pair_kernel(float* x, const T* __restrict__ y1, const float* __restrict__ w1, const T* __restrict__ y2,
                         const float* __restrict__ w2, float factor, float eps, int width, RowNext nx) {
  __shared__ float scratch[32];
  __shared__ float2 s_pair[kPairThreads / 32];
  const size_t row = blockIdx.x;
  y1 += row * width;
  y2 += row * width;
  float* xr = x + row * width;
  auto factors = [&](float ss1, float ss2) {           // both root mean squares in one meeting
    ss1 = warp_sum(ss1);
    ss2 = warp_sum(ss2);
    if ((threadIdx.x & 31) == 0) s_pair[threadIdx.x >> 5] = make_float2(ss1, ss2);
    __syncthreads();
    float2 t = make_float2(0.f, 0.f);
#pragma unroll
    for (int w = 0; w < kPairThreads / 32; ++w) { t.x += s_pair[w].x; t.y += s_pair[w].y; }
    return make_float2(factor / sqrtf(t.x / static_cast<float>(width) + eps), factor / sqrtf(t.y / static_cast<float>(width) + eps));
  };
  if constexpr (HELD) {
    float a[kPairPieces][VEC], b[kPairPieces][VEC], s[kPairPieces][VEC], ss1 = 0.f, ss2 = 0.f;
#pragma unroll
    for (int k = 0; k < kPairPieces; ++k) {
      const int c = (k * kPairThreads + static_cast<int>(threadIdx.x)) * VEC;
      if (c < width) {
        load_vec<T, VEC>(y1 + c, a[k]);
        load_vec<T, VEC>(y2 + c, b[k]);
        load_vec<float, VEC>(xr + c, s[k]);
      }
    }
#pragma unroll
    for (int k = 0; k < kPairPieces; ++k)
      if ((k * kPairThreads + static_cast<int>(threadIdx.x)) * VEC < width)
#pragma unroll
        for (int i = 0; i < VEC; ++i) { ss1 = fmaf(a[k][i], a[k][i], ss1); ss2 = fmaf(b[k][i], b[k][i], ss2); }
    const float2 f = factors(ss1, ss2);
    float ss = 0.f;
    T* out = static_cast<T*>(nx.out) + row * width;
#pragma unroll
    for (int k = 0; k < kPairPieces; ++k) {
      const int c = (k * kPairThreads + static_cast<int>(threadIdx.x)) * VEC;
      if (c < width) {
        float u[VEC], v[VEC];
        load_vec<float, VEC>(w1 + c, u);
        load_vec<float, VEC>(w2 + c, v);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          s[k][i] += a[k][i] * f.x * u[i] + b[k][i] * f.y * v[i];
          ss = fmaf(s[k][i], s[k][i], ss);
        }
        store_vec<float, VEC>(xr + c, s[k]);
        if (nx.mode == CACHEIR_B200_NEXT_COPY) store_vec<T, VEC>(out + c, s[k]);
      }
    }
    if (nx.mode != CACHEIR_B200_NEXT_RMS) return;
    const float inv = 1.f / sqrtf(block_sum_all(ss, scratch) / static_cast<float>(width) + nx.eps);
#pragma unroll
    for (int k = 0; k < kPairPieces; ++k) {
      const int c = (k * kPairThreads + static_cast<int>(threadIdx.x)) * VEC;
      if (c < width) {
        float w[VEC];
        load_vec<float, VEC>(nx.w + c, w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) w[i] = s[k][i] * inv * w[i];
        store_vec<T, VEC>(out + c, w);
      }
    }
  } else {
    float ss1 = 0.f, ss2 = 0.f;
    for (int c = threadIdx.x * VEC; c < width; c += kPairThreads * VEC) {
      float a[VEC], b[VEC];
      load_vec<T, VEC>(y1 + c, a);
      load_vec<T, VEC>(y2 + c, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) { ss1 = fmaf(a[i], a[i], ss1); ss2 = fmaf(b[i], b[i], ss2); }
    }
    const float2 f = factors(ss1, ss2);
    finish_row<T, VEC>(xr, row, width, nx, scratch, [&](int c, float (&s)[VEC]) {
      float a[VEC], b[VEC], u[VEC], v[VEC];
      load_vec<T, VEC>(y1 + c, a);
      load_vec<T, VEC>(y2 + c, b);
      load_vec<float, VEC>(w1 + c, u);
      load_vec<float, VEC>(w2 + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) s[i] += a[i] * f.x * u[i] + b[i] * f.y * v[i];
    });
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kRowThreads)
gated_rms_kernel(const T* __restrict__ o, const T* __restrict__ gate, long long gate_stride, const float* __restrict__ w, float eps,
                 T* __restrict__ out, int cols) {
  __shared__ float scratch[32];
  const size_t row = blockIdx.x;
  const T* orow = o + row * cols;
  const T* grow = gate + row * gate_stride;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < cols; c += kRowThreads * VEC) {
    float v[VEC];
    load_vec<T, VEC>(orow + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, scratch) / static_cast<float>(cols) + eps);
  for (int c = threadIdx.x * VEC; c < cols; c += kRowThreads * VEC) {
    float v[VEC], wv[VEC], g[VEC];
    load_vec<T, VEC>(orow + c, v);
    load_vec<T, VEC>(grow + c, g);
    load_vec<float, VEC>(w + c, wv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * inv * wv[i] * sigmoid_exact(g[i]);
    store_vec<T, VEC>(out + row * cols + c, v);
  }
}

// A unit is one part of one row; WARPS warps share it (one: eight units per block).
template <typename T, int VEC, int WARPS>
__global__ void __launch_bounds__(WARPS == 1 ? 256 : WARPS * 32)
gated_parts_rms_kernel(const T* __restrict__ o, const T* __restrict__ gate, long long gate_stride, const float* __restrict__ w, int shared_weight,
                       int gate_first, float eps, T* __restrict__ out, int units, int parts, int size) {
  __shared__ float scratch[32];
  const int unit = WARPS == 1 ? blockIdx.x * 8 + static_cast<int>(threadIdx.x >> 5) : static_cast<int>(blockIdx.x);
  const int at = WARPS == 1 ? static_cast<int>(threadIdx.x & 31) : static_cast<int>(threadIdx.x);
  if (unit >= units) return;
  const int row = unit / parts, part = unit % parts;
  const T* src = o + static_cast<size_t>(unit) * size;
  const T* g = gate + static_cast<size_t>(row) * gate_stride + static_cast<size_t>(part) * size;
  const float* weight = w + (shared_weight ? 0 : static_cast<size_t>(part) * size);
  T* dst = out + static_cast<size_t>(unit) * size;
  constexpr int kStep = 32 * WARPS * VEC, N = 4;      // pieces that stay in registers, requested before the sum
  auto total = [&](float ss) { return WARPS == 1 ? warp_sum(ss) : block_sum_all(ss, scratch); };
  auto gated = [&](float (&x)[VEC], const float (&gt)[VEC], float& ss) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      if (gate_first) x[i] *= silu_exact(gt[i]);
      ss = fmaf(x[i], x[i], ss);
    }
  };
  auto finish = [&](float (&x)[VEC], const float (&gt)[VEC], const float (&wv)[VEC], float inv) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] = x[i] * inv * wv[i] * (gate_first ? 1.f : silu_exact(gt[i]));
  };
  float ss = 0.f;
  if (size <= kStep * N) {
    float x[N][VEC], gt[N][VEC];
#pragma unroll
    for (int k = 0; k < N; ++k) {
      const int c = k * kStep + at * VEC;
      if (c < size) {
        load_vec<T, VEC>(src + c, x[k]);
        load_vec<T, VEC>(g + c, gt[k]);
      }
    }
#pragma unroll
    for (int k = 0; k < N; ++k)
      if (k * kStep + at * VEC < size) gated(x[k], gt[k], ss);
    const float inv = 1.f / sqrtf(total(ss) / static_cast<float>(size) + eps);
#pragma unroll
    for (int k = 0; k < N; ++k) {
      const int c = k * kStep + at * VEC;
      if (c < size) {
        float wv[VEC];
        load_vec<float, VEC>(weight + c, wv);
        finish(x[k], gt[k], wv, inv);
        store_vec<T, VEC>(dst + c, x[k]);
      }
    }
    return;
  }
  for (int c = at * VEC; c < size; c += kStep) {
    float x[VEC], gt[VEC];
    load_vec<T, VEC>(src + c, x);
    load_vec<T, VEC>(g + c, gt);
    gated(x, gt, ss);
  }
  const float inv = 1.f / sqrtf(total(ss) / static_cast<float>(size) + eps);
  for (int c = at * VEC; c < size; c += kStep) {
    float x[VEC], gt[VEC], wv[VEC], unused = 0.f;
    load_vec<T, VEC>(src + c, x);
    load_vec<T, VEC>(g + c, gt);
    load_vec<float, VEC>(weight + c, wv);
    gated(x, gt, unused);
    finish(x, gt, wv, inv);
    store_vec<T, VEC>(dst + c, x);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
glu_pairs_kernel(const T* __restrict__ y, T* __restrict__ out, int ff, int epilogue, float limit) {
  const size_t row = blockIdx.x;
  for (int c = blockIdx.y * 256 + threadIdx.x; c < ff; c += gridDim.y * 256) {
    const T* p = y + row * 2 * ff + 2 * c;
    const float a = Elem<T>::ld(p), u = Elem<T>::ld(p + 1);
    Elem<T>::st(out + row * ff + c, epilogue == CACHEIR_B200_DENSE_GEGLU ? gelu_tanh(a) * u
                                    : epilogue == CACHEIR_B200_DENSE_SWIGLU ? silu_exact(a) * u : clamped_glu(a, u, limit));
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
gelu_embed_kernel(const T* __restrict__ g, const int64_t* __restrict__ ids, const T* __restrict__ table, long long table_stride,
                  int table_col, T* __restrict__ out, int dim, int vocab) {
  const size_t row = blockIdx.x;
  const int64_t id = min(max(ids[row], static_cast<int64_t>(0)), static_cast<int64_t>(vocab - 1));
  for (int c = threadIdx.x; c < dim; c += 256)
    Elem<T>::st(out + row * dim + c, gelu_tanh(Elem<T>::ld(g + row * dim + c)) * Elem<T>::ld(table + id * table_stride + table_col + c));
}

template <typename T, bool RELU2>
__global__ void __launch_bounds__(256)
activate_cols_kernel(T* __restrict__ y, long long stride, int cols) {
  T* yr = y + static_cast<size_t>(blockIdx.x) * stride;
  for (int c = blockIdx.y * 256 + threadIdx.x; c < cols; c += gridDim.y * 256) {
    const float z = Elem<T>::ld(yr + c);
    Elem<T>::st(yr + c, RELU2 ? relu_squared(z) : silu_exact(z));
  }
}

// ---- plain tiled GEMM, float32 arithmetic: 64 tokens x 64 columns per CTA, 16 k at a time ---------------------------
constexpr int kTile = 64, kTileK = 16;
template <typename T, typename TY>
__global__ void __launch_bounds__(256)
dense_simple_kernel(const T* __restrict__ x, const T* __restrict__ w, TY* __restrict__ y, int rows, int N, int K, int w_batch_rows,
                    int x_batch_cols, int y_batch_cols, long long ws, long long xs, long long ys, const float* __restrict__ bias) {
  __shared__ float sx[kTileK][kTile + 4], sw[kTileK][kTile + 4];
  const int z = blockIdx.z;
  x += static_cast<long long>(z) * x_batch_cols;
  w += static_cast<long long>(z) * w_batch_rows * ws;
  y += static_cast<long long>(z) * y_batch_cols;
  const int t0 = blockIdx.y * kTile, n0 = blockIdx.x * kTile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kTileK) {
    for (int i = threadIdx.x; i < kTile * kTileK; i += 256) {
      const int r = i / kTileK, k = i % kTileK;
      sx[k][r] = (t0 + r < rows && k0 + k < K) ? Elem<T>::ld(x + (t0 + r) * xs + k0 + k) : 0.f;
      sw[k][r] = (n0 + r < N && k0 + k < K) ? Elem<T>::ld(w + (n0 + r) * ws + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kTileK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sx[k][ty * 4 + i]; b[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (t < rows && n < N) Elem<TY>::st(y + t * ys + n, acc[i][j] + (bias ? bias[n] : 0.f));
    }
}

// grid.y so that a small batch still spreads over the SMs
inline dim3 row_grid(int rows, int cols) {
  int y = 1;
  while (rows * y < kNumSMs * 2 && y * 256 < cols) ++y;
  return dim3(rows, y);
}
bool next_ok(int mode, const float* w, const float* b, const void* out) {
  if (mode == CACHEIR_B200_NEXT_NONE) return true;
  if (mode == CACHEIR_B200_NEXT_COPY) return out != nullptr;
  return mode == CACHEIR_B200_NEXT_DYT && w && b && out;
}

}  // namespace
}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_scaled_embedding(const void* table, const int64_t* ids, float* residual, int rows, int width, int vocab,
                                             float scale, int accumulate, int next_mode, const float* next_w, const float* next_b, float next_alpha,
                                             void* next_out, int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!table || !ids || !residual || vocab <= 0) return CACHEIR_B200_EINVAL;
  if (accumulate || row_next_norms(next_mode)) {
    if (!row_next_ok(next_mode, next_w, next_out)) return CACHEIR_B200_EINVAL;
    const RowNext rn{next_mode, next_w, next_alpha, next_out};
    const bool vec = width % 4 == 0 && aligned_to(table, 16) && aligned_to(residual, 16) && row_next_aligned(next_mode, next_w, next_out);
#define CB200_ROWS(VEC, ADD)                                                                  \
  embedding_rows_kernel<T, VEC, ADD><<<rows, kRowThreads, 0, as_stream(stream)>>>(static_cast<const T*>(table), ids, residual, width, vocab, scale, rn)
    CB200_HYBRID_DTYPE(dtype, {
      if (vec && accumulate) CB200_ROWS(4, true);
      else if (vec) CB200_ROWS(4, false);
      else if (accumulate) CB200_ROWS(1, true);
      else CB200_ROWS(1, false);
    });
#undef CB200_ROWS
    return launch_status();
  }
  if (!next_ok(next_mode, next_w, next_b, next_out)) return CACHEIR_B200_EINVAL;
  const NextArgs nx{next_mode, next_w, next_b, next_alpha, next_out};
  CB200_HYBRID_DTYPE(dtype, (scaled_embedding_kernel<T><<<row_grid(rows, width), 256, 0, as_stream(stream)>>>(
                                static_cast<const T*>(table), ids, residual, width, vocab, scale, nx)));
  return launch_status();
}

extern "C" int cacheir_b200_dyt_rows(const float* residual, const int32_t* row_index, const float* w, const float* b, float alpha,
                                     void* out, int rows, int width, int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !w || !b || !out) return CACHEIR_B200_EINVAL;
  CB200_HYBRID_DTYPE(dtype, (dyt_rows_kernel<T><<<row_grid(rows, width), 256, 0, as_stream(stream)>>>(
                                residual, row_index, w, b, alpha, static_cast<T*>(out), width)));
  return launch_status();
}

extern "C" int cacheir_b200_rms_rows(const float* residual, const int32_t* row_index, const float* w, float eps, void* out, int rows,
                                     int width, int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !w || !out) return CACHEIR_B200_EINVAL;
  const bool vec = width % 4 == 0 && aligned_to(residual, 16) && aligned_to(w, 16) && aligned_to(out, 16);
  CB200_HYBRID_DTYPE(dtype, {
    if (vec) rms_rows_kernel<T, 4><<<rows, 512, 0, as_stream(stream)>>>(residual, row_index, w, eps, static_cast<T*>(out), width);
    else rms_rows_kernel<T, 1><<<rows, 512, 0, as_stream(stream)>>>(residual, row_index, w, eps, static_cast<T*>(out), width);
  });
  return launch_status();
}

extern "C" int cacheir_b200_residual_dyt(float* residual, const void* y, const float* w, const float* b, float alpha, int rows,
                                         int width, int next_mode, const float* next_w, const float* next_b, float next_alpha,
                                         void* next_out, int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !y || !w || !b || !next_ok(next_mode, next_w, next_b, next_out)) return CACHEIR_B200_EINVAL;
  const NextArgs nx{next_mode, next_w, next_b, next_alpha, next_out};
  CB200_HYBRID_DTYPE(dtype, (residual_dyt_kernel<T><<<row_grid(rows, width), 256, 0, as_stream(stream)>>>(
                                residual, static_cast<const T*>(y), w, b, alpha, width, nx)));
  return launch_status();
}

extern "C" int cacheir_b200_layer_norm_rows(const float* residual, const int32_t* row_index, const float* w, float eps, void* out, int rows,
                                            int width, int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !w || !out) return CACHEIR_B200_EINVAL;
  const bool vec = width % 4 == 0 && aligned_to(residual, 16) && aligned_to(w, 16) && aligned_to(out, 16);
  CB200_HYBRID_DTYPE(dtype, {
    if (vec) layer_norm_rows_kernel<T, 4><<<rows, 512, 0, as_stream(stream)>>>(residual, row_index, w, eps, static_cast<T*>(out), width);
    else layer_norm_rows_kernel<T, 1><<<rows, 512, 0, as_stream(stream)>>>(residual, row_index, w, eps, static_cast<T*>(out), width);
  });
  return launch_status();
}

extern "C" int cacheir_b200_join_embedding(const float* residual, const void* table, const int64_t* ids, void* out, int rows, int width, int vocab,
                                           int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !table || !ids || !out || vocab <= 0) return CACHEIR_B200_EINVAL;
  const bool vec = width % 4 == 0 && aligned_to(residual, 16) && aligned_to(table, 16) && aligned_to(out, 16);
  CB200_HYBRID_DTYPE(dtype, {
    if (vec) join_embedding_kernel<T, 4><<<row_grid(rows, width / 4), 256, 0, as_stream(stream)>>>(
        residual, static_cast<const T*>(table), ids, static_cast<T*>(out), width, vocab);
    else join_embedding_kernel<T, 1><<<row_grid(rows, width), 256, 0, as_stream(stream)>>>(
        residual, static_cast<const T*>(table), ids, static_cast<T*>(out), width, vocab);
  });
  return launch_status();
}

extern "C" int cacheir_b200_residual_add(float* residual, const void* y, const float* scale, int rows, int width, int next_mode, const float* next_w,
                                         const float* next_b, float next_alpha, void* next_out, int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !y || next_b || !row_next_ok(next_mode, next_w, next_out)) return CACHEIR_B200_EINVAL;
  const RowNext nx{next_mode, next_w, next_alpha, next_out};
  const bool vec = width % 4 == 0 && aligned_to(residual, 16) && aligned_to(y, 16) && (!scale || aligned_to(scale, 16)) &&
                   row_next_aligned(next_mode, next_w, next_out);
#define CB200_ADD(VEC, HELD) \
  residual_add_kernel<T, VEC, HELD><<<rows, kAddThreads, 0, as_stream(stream)>>>(residual, static_cast<const T*>(y), scale, width, nx)
  CB200_HYBRID_DTYPE(dtype, {
    if (vec && width <= 4 * kAddThreads * kAddPieces) CB200_ADD(4, true);
    else if (vec) CB200_ADD(4, false);
    else CB200_ADD(1, false);
  });
#undef CB200_ADD
  return launch_status();
}

extern "C" int cacheir_b200_residual_rms_pair(float* residual, const void* y1, const float* w1, const void* y2, const float* w2, float factor,
                                              float eps, int rows, int width, int next_mode, const float* next_w, const float* next_b,
                                              float next_alpha, void* next_out, int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !y1 || !w1 || !y2 || !w2 || next_b || !row_next_ok(next_mode, next_w, next_out)) return CACHEIR_B200_EINVAL;
  const RowNext nx{next_mode, next_w, next_alpha, next_out};
  const bool vec = width % 4 == 0 && aligned_to(residual, 16) && aligned_to(y1, 16) && aligned_to(y2, 16) && aligned_to(w1, 16) &&
                   aligned_to(w2, 16) && row_next_aligned(next_mode, next_w, next_out);
#define CB200_PAIR(VEC, HELD)                                                                                                        \
  residual_rms_pair_kernel<T, VEC, HELD><<<rows, kPairThreads, 0, as_stream(stream)>>>(residual, static_cast<const T*>(y1), w1,        \
                                                                                      static_cast<const T*>(y2), w2, factor, eps, width, nx)
  CB200_HYBRID_DTYPE(dtype, {
    if (vec && width <= 4 * kPairThreads * kPairPieces && next_mode != CACHEIR_B200_NEXT_LAYER) CB200_PAIR(4, true);
    else if (vec) CB200_PAIR(4, false);
    else CB200_PAIR(1, false);
  });
#undef CB200_PAIR
  return launch_status();
}

extern "C" int cacheir_b200_residual_rms(float* residual, const void* y, const float* w, float eps, int rows, int width,
                                         int next_mode, const float* next_w, const float* next_b, float next_alpha, void* next_out,
                                         int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (!residual || !y || !w || !next_ok(next_mode, next_w, next_b, next_out)) return CACHEIR_B200_EINVAL;
  const NextArgs nx{next_mode, next_w, next_b, next_alpha, next_out};
  const bool vec = width % 4 == 0 && aligned_to(residual, 16) && aligned_to(y, 16) && aligned_to(w, 16) &&
                   (next_mode == CACHEIR_B200_NEXT_NONE || aligned_to(next_out, 16)) &&
                   (next_mode != CACHEIR_B200_NEXT_DYT || (aligned_to(next_w, 16) && aligned_to(next_b, 16)));
  CB200_HYBRID_DTYPE(dtype, {
    if (vec) residual_rms_kernel<T, 4><<<rows, kRowThreads, 0, as_stream(stream)>>>(residual, static_cast<const T*>(y), w, eps, width, nx);
    else residual_rms_kernel<T, 1><<<rows, kRowThreads, 0, as_stream(stream)>>>(residual, static_cast<const T*>(y), w, eps, width, nx);
  });
  return launch_status();
}

extern "C" int cacheir_b200_gated_rms(const void* o, const void* gate, long long gate_stride, const float* w, float eps, void* out,
                                      int rows, int cols, int dtype, void* stream) {
  if (rows <= 0 || cols <= 0) return 0;
  if (!o || !gate || !w || !out) return CACHEIR_B200_EINVAL;
  const bool vec = cols % 4 == 0 && gate_stride % 4 == 0 && aligned_to(o, 16) && aligned_to(gate, 16) && aligned_to(w, 16) && aligned_to(out, 16);
  CB200_HYBRID_DTYPE(dtype, {
    if (vec) gated_rms_kernel<T, 4><<<rows, kRowThreads, 0, as_stream(stream)>>>(
        static_cast<const T*>(o), static_cast<const T*>(gate), gate_stride, w, eps, static_cast<T*>(out), cols);
    else gated_rms_kernel<T, 1><<<rows, kRowThreads, 0, as_stream(stream)>>>(
        static_cast<const T*>(o), static_cast<const T*>(gate), gate_stride, w, eps, static_cast<T*>(out), cols);
  });
  return launch_status();
}

extern "C" int cacheir_b200_glu_pairs(const void* y, void* out, int rows, int ff, int epilogue, float limit, int dtype, void* stream) {
  if (rows <= 0 || ff <= 0) return 0;
  if (!y || !out || (epilogue != CACHEIR_B200_DENSE_GEGLU && epilogue != CACHEIR_B200_DENSE_SWIGLU && epilogue != CACHEIR_B200_DENSE_CLAMPED_GLU))
    return CACHEIR_B200_EINVAL;
  CB200_HYBRID_DTYPE(dtype, (glu_pairs_kernel<T><<<row_grid(rows, ff), 256, 0, as_stream(stream)>>>(
                                static_cast<const T*>(y), static_cast<T*>(out), ff, epilogue, limit)));
  return launch_status();
}

extern "C" int cacheir_b200_gelu_embed(const void* g, const int64_t* ids, const void* table, long long table_stride, int table_col,
                                       void* out, int rows, int dim, int vocab, int dtype, void* stream) {
  if (rows <= 0 || dim <= 0) return 0;
  if (!g || !ids || !table || !out || vocab <= 0) return CACHEIR_B200_EINVAL;
  CB200_HYBRID_DTYPE(dtype, (gelu_embed_kernel<T><<<rows, 256, 0, as_stream(stream)>>>(
                                static_cast<const T*>(g), ids, static_cast<const T*>(table), table_stride, table_col,
                                static_cast<T*>(out), dim, vocab)));
  return launch_status();
}

extern "C" int cacheir_b200_silu_cols(void* y, int rows, long long stride, int cols, int dtype, void* stream) {
  if (rows <= 0 || cols <= 0) return 0;
  if (!y) return CACHEIR_B200_EINVAL;
  CB200_HYBRID_DTYPE(dtype, (activate_cols_kernel<T, false><<<row_grid(rows, cols), 256, 0, as_stream(stream)>>>(static_cast<T*>(y), stride, cols)));
  return launch_status();
}

extern "C" int cacheir_b200_relu2_cols(void* y, int rows, long long stride, int cols, int dtype, void* stream) {
  if (rows <= 0 || cols <= 0) return 0;
  if (!y) return CACHEIR_B200_EINVAL;
  CB200_HYBRID_DTYPE(dtype, (activate_cols_kernel<T, true><<<row_grid(rows, cols), 256, 0, as_stream(stream)>>>(static_cast<T*>(y), stride, cols)));
  return launch_status();
}

extern "C" int cacheir_b200_gated_parts_rms(const void* o, const void* gate, long long gate_stride, const float* w, int shared_weight,
                                            int gate_first, float eps, void* out, int rows, int cols, int parts, int dtype, void* stream) {
  if (rows <= 0 || cols <= 0) return 0;
  if (!o || !gate || !w || !out || parts <= 0 || cols % parts != 0) return CACHEIR_B200_EINVAL;
  const int size = cols / parts, units = rows * parts, quad = 4 * (dtype == CACHEIR_B200_F32 ? 4 : 2);
  const bool vec = size % 4 == 0 && gate_stride % 4 == 0 && aligned_to(o, quad) && aligned_to(gate, quad) && aligned_to(w, 16) && aligned_to(out, quad);
#define CB200_PARTS(VEC, WARPS)                                                                                                         \
  gated_parts_rms_kernel<T, VEC, WARPS><<<WARPS == 1 ? (units + 7) / 8 : units, WARPS == 1 ? 256 : WARPS * 32, 0, as_stream(stream)>>>(                             \
      static_cast<const T*>(o), static_cast<const T*>(gate), gate_stride, w, shared_weight, gate_first, eps, static_cast<T*>(out), units, parts, size)
  CB200_HYBRID_DTYPE(dtype, {
    if (vec && size <= 512) CB200_PARTS(4, 1);
    else if (vec && size <= 1024) CB200_PARTS(4, 2);
    else if (vec) CB200_PARTS(4, 8);
    else if (size <= 512) CB200_PARTS(1, 1);
    else CB200_PARTS(1, 8);
  });
#undef CB200_PARTS
  return launch_status();
}

extern "C" int cacheir_b200_dense_simple(const void* x, const void* w, void* y, int rows, int N, int K, int batch, int w_batch_rows,
                                         int x_batch_cols, int y_batch_cols, long long w_stride, long long x_stride,
                                         long long y_stride, const float* bias, int dtype, int y_dtype, void* stream) {
  if (rows <= 0 || N <= 0) return 0;
  if (K <= 0 || !x || !w || !y || batch < 1 || (batch > 1 && bias)) return CACHEIR_B200_EINVAL;
  const dim3 grid((N + kTile - 1) / kTile, (rows + kTile - 1) / kTile, batch);
  if (grid.y > 65535 || grid.z > 65535) return CACHEIR_B200_ELIMIT;
  cudaStream_t st = as_stream(stream);
#define CB200_SIMPLE(T, TY)                                                                                              \
  dense_simple_kernel<T, TY><<<grid, 256, 0, st>>>(static_cast<const T*>(x), static_cast<const T*>(w), static_cast<TY*>(y), rows, N, \
                                                   K, w_batch_rows, x_batch_cols, y_batch_cols, w_stride, x_stride, y_stride, bias)
  if (dtype == CACHEIR_B200_F32 && y_dtype == CACHEIR_B200_F32) CB200_SIMPLE(float, float);
  else if (dtype == CACHEIR_B200_BF16 && y_dtype == CACHEIR_B200_F32) CB200_SIMPLE(__nv_bfloat16, float);
  else if (dtype == CACHEIR_B200_BF16 && y_dtype == CACHEIR_B200_BF16) CB200_SIMPLE(__nv_bfloat16, __nv_bfloat16);
  else return CACHEIR_B200_EUNSUPPORTED;
#undef CB200_SIMPLE
  return launch_status();
}
