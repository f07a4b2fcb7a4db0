// What the kernels of tied attention share: the pages a step reads, the cap on scores, the cache's tensor map.
#pragma once

#include "cacheir_b200_experts.h"
#include "hybrid_common.cuh"
#include "tc_ptx.cuh"

namespace cb200 {

constexpr int kTiedPage = 64;                    // cache rows of a page in the tensor-core kernels
constexpr int kTiedBox = kTiedPage * 128;        // 64 rows x 64 columns, 128-byte swizzle
constexpr float kLog2e = 1.4426950408889634f;

// Columns of a cached row that prepared queries leave out: whole 64-column boxes of which they would be zero.
__host__ __device__ inline int tied_lead(int key_from) { return key_from / 64 * 64; }

__device__ __forceinline__ float tied_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// score * log2 e from the raw product. tanh(x) = 1 - 2 / (1 + e^2x): the error of exponential and quotient stays near
// 2^-22 of the cap, also where the score is small.
struct TiedScore {
  float pre, cap2;      // factor of the raw product; cap * log2 e, 0 without a cap
  __device__ __forceinline__ float operator()(float raw) const {
    if (cap2 == 0.f) return raw * pre;
    return cap2 - __fdividef(2.f * cap2, 1.f + tied_ex2(raw * pre));
  }
};
inline TiedScore tied_score(float scale, float cap) {
  if (cap > 0.f) return {scale * 2.f * kLog2e / cap, cap * kLog2e};
  return {scale * kLog2e, 0.f};
}

// The pages that rows at positions pos0.. see: the kept first ones, then the window's.
struct TiedPages {
  int kept, page_lo, total;
  __device__ __forceinline__ TiedPages(const cacheir_b200_tied_args& a, int pos0, int pos_last) {
    page_lo = max(0, pos0 - a.window + 1) / a.page_size;
    kept = min((a.keep_first + a.page_size - 1) / a.page_size, page_lo);
    total = kept + pos_last / a.page_size - page_lo + 1;
  }
  __device__ __forceinline__ int page(int it) const { return it < kept ? it : page_lo + it - kept; }
};

__device__ __forceinline__ int tied_slot(const cacheir_b200_tied_args& a, int seg, int page) {
  const int slot = page < a.max_pages ? a.page_table[static_cast<size_t>(seg) * a.max_pages + page] : 0;
  return min(max(slot, 0), a.num_slots - 1);
}

inline bool tied_encode(CUtensorMap* map, const void* base, uint64_t width, uint64_t rows) {
  ptx::EncodeTiledFn fn = ptx::tensor_map_encoder();
  if (!fn) return false;
  const cuuint64_t dims[2] = {width, rows};
  const cuuint64_t strides[1] = {width * 2};
  const cuuint32_t box[2] = {64, kTiedPage};
  const cuuint32_t elem_strides[2] = {1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem_strides,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

inline bool tied_args_ok(const cacheir_b200_tied_args& a) {
  return a.positions && a.row_seg && a.page_table && a.pool && a.inv_rms && a.segments > 0 && a.max_pages > 0 && a.page_size > 0 &&
         a.num_slots > 0 && a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.dim <= a.width && a.key_from >= 0 &&
         a.key_from < a.width && a.window > 0 && a.keep_first >= 0 && a.heads <= 65535;
}

}  // namespace cb200
