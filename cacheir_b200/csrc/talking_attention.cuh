// What the kernels of talking-heads attention share.
#pragma once

#include "cacheir_b200_talking.h"
#include "hybrid_common.cuh"
#include "tc_ptx.cuh"

namespace cb200 {

constexpr int kTalkPage = 64;                    // cache rows of a page in the tensor-core kernels
constexpr float kTalkLog2e = 1.4426950408889634f;

__device__ __forceinline__ float talk_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ int talk_slot(const cacheir_b200_talking_args& a, int seg, int page) {
  const int slot = page < a.max_pages ? a.page_table[static_cast<size_t>(seg) * a.max_pages + page] : 0;
  return min(max(slot, 0), a.num_slots - 1);
}

// cached rows as boxes of 64 columns (128-byte swizzle) and `box_rows` rows
inline bool talk_encode(CUtensorMap* map, const void* base, uint64_t width, uint64_t rows, uint32_t box_rows) {
  ptx::EncodeTiledFn fn = ptx::tensor_map_encoder();
  if (!fn) return false;
  const cuuint64_t dims[2] = {width, rows};
  const cuuint64_t strides[1] = {width * 2};
  const cuuint32_t box[2] = {64, box_rows};
  const cuuint32_t elem_strides[2] = {1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem_strides,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

inline bool talk_args_ok(const cacheir_b200_talking_args& a) {
  return a.positions && a.row_seg && a.page_table && a.keys && a.values && a.talk && a.segments > 0 && a.max_pages > 0 && a.page_size > 0 &&
         a.num_slots > 0 && a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.vdim > 0 && a.window > 0 && a.heads <= 65535;
}

int talking_prompt_status(bool reset);

}  // namespace cb200
