// Shared by the kernels of the hybrid decoder families (latent attention, linear recurrences, Dynamic Tanh layers).
#pragma once

#include "cacheir_b200_hybrid.h"
#include "common.cuh"

namespace cb200 {

// These families bound their logits against 32-bit arithmetic, so activations use the accurate expf / tanhf.
__device__ __forceinline__ float sigmoid_exact(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_exact(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float gelu_tanh(float z) {
  constexpr float kRoot2OverPi = 0.7978845608028654f;
  return 0.5f * z * (1.f + tanhf(kRoot2OverPi * fmaf(0.044715f * z * z, z, z)));
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

}  // namespace cb200
