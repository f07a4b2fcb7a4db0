// Shared by the kernels of the hybrid decoder families (latent attention, linear recurrences, Dynamic Tanh layers).
#pragma once

#include "cacheir_b200_ragged.h"
#include "common.cuh"

namespace cb200 {

// These families bound their logits against 32-bit arithmetic, so activations use the accurate expf / tanhf. The quotient
// (2 ulp) has no slow path to branch to, so that a thread's many elements overlap; past the exponential's range it is 0.
__device__ __forceinline__ float sigmoid_exact(float z) { return __fdividef(1.f, 1.f + expf(-z)); }
__device__ __forceinline__ float silu_exact(float z) { return z * sigmoid_exact(z); }
__device__ __forceinline__ float relu_squared(float z) { return z > 0.f ? z * z : 0.f; }
__device__ __forceinline__ float gelu_tanh(float z) {
  constexpr float kRoot2OverPi = 0.7978845608028654f;
  return 0.5f * z * (1.f + tanhf(kRoot2OverPi * fmaf(0.044715f * z * z, z, z)));
}

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ float clamped_glu(float gate, float up, float limit) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g * sigmoid_exact(1.702f * g) * (u + 1.f);
}

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }

// sum over a block of up to 32 warps; every thread gets the result
__device__ __forceinline__ float block_sum_all(float v, float* scratch) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < static_cast<int>((blockDim.x + 31) >> 5); ++w) t += scratch[w];
  return t;
}

// bf16 warp MMA pieces (16x8x16, fp32 accumulation)
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x2(uint32_t addr, uint32_t (&r)[2]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
// v = hi + lo with both halves bf16: a product with either half on the tensor cores keeps v to about 2^-17
__device__ __forceinline__ void split_bf16(float v, float* hi, float* lo) {
  *hi = __bfloat162float(__float2bfloat16_rn(v));
  *lo = v - *hi;
}

// VEC neighbouring elements per access
template <typename T, int VEC>
__device__ __forceinline__ void load_vec(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(T) == 2) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(raw.x << 16); v[1] = __uint_as_float(raw.x & 0xffff0000u);
    v[2] = __uint_as_float(raw.y << 16); v[3] = __uint_as_float(raw.y & 0xffff0000u);
  } else if constexpr (VEC == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    v[0] = Elem<T>::ld(p);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(T) == 2) {
    uint2 raw;
    raw.x = pack_bf16(v[0], v[1]);
    raw.y = pack_bf16(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = raw;
  } else if constexpr (VEC == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    Elem<T>::st(p, v[0]);
  }
}

// reads a kernel's status word (a __device__ int), clearing it on request; synchronises
template <typename Symbol>
int device_status_word(Symbol& word, bool reset) {
  int status = 0;
  if (cudaMemcpyFromSymbol(&status, word, sizeof(int)) != cudaSuccess) return -1;
  if (reset && status != 0) {
    const int zero = 0;
    cudaMemcpyToSymbol(word, &zero, sizeof(int));
  }
  return status;
}

}  // namespace cb200

// runs a statement with T = the activation type
#define CB200_HYBRID_DTYPE(dtype, ...)                                                  \
  switch (dtype) {                                                                      \
    case CACHEIR_B200_F32: { using T = float; __VA_ARGS__; break; }                     \
    case CACHEIR_B200_BF16: { using T = __nv_bfloat16; __VA_ARGS__; break; }            \
    default: return CACHEIR_B200_EUNSUPPORTED;                                          \
  }
