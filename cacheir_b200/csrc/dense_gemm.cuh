// Dense bf16 GEMM on the 5th-generation tensor cores with elementwise epilogues, sm_100a.
//
//   Y[t, n] = f( sum_k X[t, k] W[n, k] )        X [T, K], W [N, K] bf16, fp32 accumulation
//
// The weight tile is the 128-row MMA operand, the token tile (16 to 256 rows) the other one, so a decode batch and a
// prompt use the same kernel and the accumulator has one weight row per tensor-memory lane: an epilogue thread owns an
// output column, keeps that column's norm constants in registers, and 32 lanes store 32 neighbouring outputs.
//
//   warp 0      TMA producer: a 64-column k block of W and X per ring stage (128-byte swizzle; what lies outside the
//               tensors reads as zero, so K needs no padding beyond the 16-byte row rule)
//   warp 1      one thread issues tcgen05.mma (M 128, N = token tile, K 16; four per stage)
//   warps 2..9  epilogue: tensor memory -> registers -> f -> global; lane quarter = warp % 4, two warps per quarter
//
// Few tiles: the K range is split over the CTAs of a cluster. Each leaves its fp32 partials in its drained ring, and
// rank r adds the partials of its share of the tokens in rank order through distributed shared memory.
// Because Dynamic Tanh is elementwise, one epilogue finishes a whole sublayer boundary: y -> norm -> residual add
// (32-bit) -> the next norm's output as the next GEMM's bf16 operand.
// `batch` > 1 runs one GEMM per head: head z takes W rows z*w_batch_rows.. and X columns z*x_batch_cols...
// GROUPED runs one GEMM per expert over the places [cu[e], cu[e+1]) of a routed step: a token tile belongs to one expert
// (found from cu on the device) and takes W rows e*w_batch_rows... X rows are places; or, with place_of, the step's rows
// themselves: an expert multiplies all of them (at most a tile, and the weights are what takes the time) and keeps those
// that chose it.
#pragma once

#include "hybrid_common.cuh"
#include "ragged.cuh"
#include "tc_ptx.cuh"

namespace cb200 {
namespace {

using namespace ptx;

constexpr int kTileN = 128;
constexpr int kBlockK = 64;               // elements of k per stage: one 128-byte swizzle span
constexpr int kWBytes = kTileN * kBlockK * 2;
constexpr int kThreads = 320;
constexpr int kTailBytes = 512;                    // barriers; from byte 128 on the places of up to 64 rows

__device__ int g_dense_status = 0;

__host__ __device__ constexpr int stage_bytes(int mt) { return kWBytes + mt * kBlockK * 2; }
__host__ __device__ constexpr int num_stages(int mt) {
  return mt <= 16 ? 5 : mt <= 64 ? 4 : mt == 128 ? 3 : 4;      // up to 128 tokens: two CTAs per SM
}
__host__ __device__ constexpr int ctas_per_sm(int mt) { return mt <= 128 ? 2 : 1; }
__host__ __device__ constexpr int tmem_cols(int mt) { return mt < 32 ? 32 : mt; }

__device__ __forceinline__ void mma_f16_ss(uint32_t tmem_d, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(tmem_d), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate) : "memory");
}
__device__ __forceinline__ void tmem_ld_x16(uint32_t taddr, float (&v)[16]) {
  uint32_t r[16];
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
        "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr) : "memory");
  tc_wait_ld();
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
}
__device__ __forceinline__ float ld_peer(uint32_t local_addr, uint32_t rank) {
  uint32_t remote;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local_addr), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
  return v;
}
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

struct Groups {
  const int32_t* cu;         // [batch + 1]
  const int32_t* place_of;   // [x_rows, top]: X rows are the step's rows; NULL: they are places
  int top, x_rows;
};

// gate and up of one unit -> its activation
template <int EPI>
__device__ __forceinline__ float paired(float g, float u, float limit) {
  if constexpr (EPI == CACHEIR_B200_DENSE_GEGLU) return gelu_tanh(g) * u;
  else if constexpr (EPI == CACHEIR_B200_DENSE_SWIGLU) return silu_exact(g) * u;
  else return clamped_glu(g, u, limit);
}
constexpr bool is_paired(int epi) {
  return epi == CACHEIR_B200_DENSE_GEGLU || epi == CACHEIR_B200_DENSE_SWIGLU || epi == CACHEIR_B200_DENSE_CLAMPED_GLU;
}

template <int EPI, int MT, bool GROUPED>
__global__ void __launch_bounds__(kThreads, ctas_per_sm(MT))
dense_gemm_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x,
                  const cacheir_b200_dense_args p, int n_tiles, const Groups groups) {
  constexpr int kStages = num_stages(MT);
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint8_t* s_w = smem;
  uint8_t* s_x = smem + kStages * kWBytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + kStages * stage_bytes(MT));
  uint64_t* full = bars;
  uint64_t* empty = bars + kStages;
  uint64_t* acc_full = empty + kStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_full + 1);

  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;
  const int split = static_cast<int>(gridDim.y);
  const int krank = static_cast<int>(blockIdx.y);      // the cluster spans the whole y extent
  int t0 = blockIdx.x * MT, t_end = p.T, z = blockIdx.z / n_tiles;
  if constexpr (GROUPED) {
    const RaggedItem it = find_item(groups.cu, p.batch, groups.place_of ? 1 << 30 : MT, blockIdx.x);
    if (it.seg < 0) return;                // (the whole cluster)
    z = it.seg; t0 = it.row0; t_end = it.row0 + it.count;
    if (groups.place_of) { t0 = 0; t_end = groups.x_rows; }
  }
  const int n0 = (blockIdx.z % n_tiles) * kTileN;
  const int kblocks_all = (p.K + kBlockK - 1) / kBlockK;
  const int kb_begin = kblocks_all * krank / split;
  const int total = kblocks_all * (krank + 1) / split - kb_begin;

  if (warp == 0 && lane == 0) {
    for (int s = 0; s < kStages; ++s) { mbar_init(smem_u32(&full[s]), 1); mbar_init(smem_u32(&empty[s]), 1); }
    mbar_init(smem_u32(acc_full), 1);
    mbar_fence_init();
  }
  if (warp == 1) tc_alloc(smem_u32(tmem_slot), tmem_cols(MT));
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  // epilogue thread: output column n of this batch entry, tokens `half`-interleaved
  const int q = warp & 3;
  const int half = (warp - 2) >> 2;
  const int r = q * 32 + lane;
  const int n = n0 + r;
  const bool n_ok = n < p.N;

  bool ok = true;
  if (warp == 0) {
    if (lane == 0) {
      int issued = 0;
      for (int i = 0; i < total; ++i) {
        const int s = i % kStages;
        if (i >= kStages && !mbar_wait(smem_u32(&empty[s]), ((i / kStages) & 1) ^ 1, &g_dense_status, (6 << 8) | 1)) break;
        const uint32_t bar = smem_u32(&full[s]);
        mbar_expect_tx(bar, stage_bytes(MT));
        const int k = (kb_begin + i) * kBlockK;
        tma_load_2d(smem_u32(s_w + s * kWBytes), &tmap_w, bar, k, z * p.w_batch_rows + n0);
        tma_load_2d(smem_u32(s_x + s * MT * kBlockK * 2), &tmap_x, bar, GROUPED ? k : z * p.x_batch_cols + k, t0);
        issued = i + 1;
      }
      if (issued < total)          // a wait gave up: nothing may still be on its way when the block ends
        for (int i = issued > kStages ? issued - kStages : 0; i < issued; ++i)
          mbar_wait(smem_u32(&full[i % kStages]), (i / kStages) & 1, &g_dense_status, (6 << 8) | 4);
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      // fp32 accumulator, bf16 x bf16, both K-major, N = MT, M = 128
      const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(MT >> 3) << 17) |
                             (static_cast<uint32_t>(kTileN >> 4) << 24);
      for (int i = 0; i < total; ++i) {
        const int s = i % kStages;
        if (!mbar_wait(smem_u32(&full[s]), (i / kStages) & 1, &g_dense_status, (6 << 8) | 2)) break;
        tc_fence_after();
        const uint32_t wb = smem_u32(s_w + s * kWBytes), xb = smem_u32(s_x + s * MT * kBlockK * 2);
#pragma unroll
        for (int j = 0; j < kBlockK / 16; ++j)
          mma_f16_ss(tmem, smem_desc_sw128(wb + j * 32), smem_desc_sw128(xb + j * 32), idesc, (i > 0 || j > 0) ? 1u : 0u);
        tc_commit(smem_u32(&empty[s]));
      }
      tc_commit(smem_u32(acc_full));
    }
    __syncwarp();
  }

  if (warp >= 2) {
    // per-column constants are requested before the wait
    float w1 = 0.f, b1 = 0.f, w2 = 0.f, b2 = 0.f;
    const float bias = (!GROUPED && p.bias && n_ok) ? p.bias[n] : 0.f;
    if (EPI == CACHEIR_B200_DENSE_RESIDUAL && n_ok) {
      w1 = p.norm_w[n]; b1 = p.norm_b[n];
      if (p.next_mode == CACHEIR_B200_NEXT_DYT) { w2 = p.next_w[n]; b2 = p.next_b[n]; }
    }
    const int* s_place = reinterpret_cast<const int*>(smem + kStages * stage_bytes(MT) + 128);
    if constexpr (GROUPED && MT <= 64) {
      if (groups.place_of) {               // where each row's result goes, if this expert has one
        const int t = threadIdx.x - 64, lo = groups.cu[z], hi = groups.cu[z + 1];
        if (t < MT) {
          int place = -1;
          if (t < t_end)
            for (int k = 0; k < groups.top; ++k) {
              const int at = groups.place_of[t * groups.top + k];
              if (at >= lo && at < hi) place = at;
            }
          const_cast<int*>(s_place)[t] = place;
        }
        asm volatile("barrier.cta.sync 2, 256;" ::: "memory");
      }
    }
    auto row_of = [&](int t) {             // output row, -1: none
      if (t >= t_end) return -1;
      if constexpr (GROUPED && MT <= 64) {
        if (groups.place_of) return s_place[t];
      }
      return t;
    };
    ok = mbar_wait(smem_u32(acc_full), 0, &g_dense_status, (6 << 8) | 3);
    tc_fence_after();
    const long long ycol = GROUPED ? n : static_cast<long long>(z) * p.y_batch_cols + n;

    auto emit = [&](auto& v, auto count, int c0) {       // v[j] = column n of token t0 + c0 + j
      constexpr int G = decltype(count)::value;
#pragma unroll
      for (int j = 0; j < G; ++j) v[j] += bias;
      if constexpr (is_paired(EPI)) {
        // W rows alternate gate, up: neighbouring lanes trade, the even lane finishes token j and the odd one j + 1
        const bool odd = (r & 1) != 0, tail = n >= p.N - p.tail_cols;      // (tail: plain float32 columns behind the pairs)
#pragma unroll
        for (int j = 0; j < G; j += 2) {
          const float got = __shfl_xor_sync(0xffffffffu, odd ? v[j] : v[j + 1], 1);
          const float y = odd ? paired<EPI>(got, v[j + 1], p.limit) : paired<EPI>(v[j], got, p.limit);
          const int row = row_of(t0 + c0 + j + (odd ? 1 : 0));
          if (n_ok && !tail && row >= 0)
            static_cast<__nv_bfloat16*>(p.y)[static_cast<long long>(row) * p.y_stride + (n >> 1)] = __float2bfloat16_rn(y);
          if (n_ok && tail) {
            float* dst = p.tail + static_cast<long long>(t0 + c0 + j) * p.tail_stride + (n - (p.N - p.tail_cols));
            if (t0 + c0 + j < t_end) dst[0] = v[j];
            if (t0 + c0 + j + 1 < t_end) dst[p.tail_stride] = v[j + 1];
          }
        }
      } else if constexpr (EPI == CACHEIR_B200_DENSE_RESIDUAL) {
        float x[G];
#pragma unroll
        for (int j = 0; j < G; ++j) {
          const int t = t0 + c0 + j;
          x[j] = (n_ok && t < t_end) ? p.residual[static_cast<long long>(t) * p.N + n] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < G; ++j) {
          const int t = t0 + c0 + j;
          if (!(n_ok && t < t_end)) continue;
          const float s = x[j] + fmaf(tanhf(p.norm_alpha * v[j]), w1, b1);
          p.residual[static_cast<long long>(t) * p.N + n] = s;
          if (p.next_mode == CACHEIR_B200_NEXT_DYT)
            static_cast<__nv_bfloat16*>(p.next_out)[static_cast<long long>(t) * p.N + n] =
                __float2bfloat16_rn(fmaf(tanhf(p.next_alpha * s), w2, b2));
          else if (p.next_mode == CACHEIR_B200_NEXT_COPY)
            static_cast<__nv_bfloat16*>(p.next_out)[static_cast<long long>(t) * p.N + n] = __float2bfloat16_rn(s);
        }
      } else {
        // what the epilogue multiplies with is loaded for all tokens before anything is stored
        float f[G];
        if constexpr (EPI == CACHEIR_B200_DENSE_GATED) {
#pragma unroll
          for (int j = 0; j < G; ++j) {
            const int t = t0 + c0 + j;
            f[j] = (n_ok && t < t_end) ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.gate)[static_cast<long long>(t) * p.gate_stride + ycol]) : 0.f;
          }
        } else if constexpr (EPI == CACHEIR_B200_DENSE_GELU_EMBED) {
          int64_t id[G];
#pragma unroll
          for (int j = 0; j < G; ++j) id[j] = p.ids[min(t0 + c0 + j, t_end - 1)];
#pragma unroll
          for (int j = 0; j < G; ++j) {
            id[j] = min(max(id[j], static_cast<int64_t>(0)), static_cast<int64_t>(p.vocab - 1));
            f[j] = n_ok ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.table)[id[j] * p.table_stride + p.table_col + n]) : 0.f;
          }
        }
#pragma unroll
        for (int j = 0; j < G; ++j) {
          const int t = row_of(t0 + c0 + j);
          if (!n_ok || t < 0) continue;
          float y = v[j];
          if constexpr (!GROUPED && (EPI == CACHEIR_B200_DENSE_BF16 || EPI == CACHEIR_B200_DENSE_SILU)) {
            if (n >= p.N - p.tail_cols) {        // plain float32 columns behind the others
              p.tail[static_cast<long long>(t) * p.tail_stride + (n - (p.N - p.tail_cols))] = y;
              continue;
            }
          }
          if constexpr (EPI == CACHEIR_B200_DENSE_F32) {
            static_cast<float*>(p.y)[static_cast<long long>(t) * p.y_stride + ycol] = y;
            continue;
          } else if constexpr (EPI == CACHEIR_B200_DENSE_SILU) {
            if (n < p.act_cols) y = silu_exact(y);
          } else if constexpr (EPI == CACHEIR_B200_DENSE_RELU2) {
            y = relu_squared(y);
          } else if constexpr (EPI == CACHEIR_B200_DENSE_GATED) {
            y *= sigmoid_exact(f[j]);
          } else if constexpr (EPI == CACHEIR_B200_DENSE_GELU_EMBED) {
            y = gelu_tanh(y) * f[j];
          }
          static_cast<__nv_bfloat16*>(p.y)[static_cast<long long>(t) * p.y_stride + ycol] = __float2bfloat16_rn(y);
        }
      }
    };

    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(q * 32) << 16);
    if (split == 1) {
      if (ok) {
        for (int c0 = half * 16; c0 < MT; c0 += 32) {
          if (t0 + c0 >= t_end) break;
          float v[16];
          tmem_ld_x16(lane_addr + c0, v);
          emit(v, std::integral_constant<int, 16>{}, c0);
        }
      }
    } else {
      float* part = reinterpret_cast<float*>(smem);            // [MT tokens][128 columns], over the drained ring
      for (int c0 = half * 16; c0 < MT; c0 += 32) {
        float v[16];
        tmem_ld_x16(lane_addr + c0, v);
#pragma unroll
        for (int j = 0; j < 16; ++j) part[(c0 + j) * kTileN + r] = v[j];
      }
      cluster_sync_all();
      const int share = MT / split;
      for (int c = krank * share + half * 2; c < (krank + 1) * share; c += 4) {
        if (t0 + c >= t_end) break;
        float v[2] = {0.f, 0.f};
        const uint32_t a = smem_u32(part + c * kTileN + r);
        for (int s = 0; s < split; ++s) {
          v[0] += ld_peer(a, s);
          v[1] += ld_peer(a + kTileN * 4, s);
        }
        emit(v, std::integral_constant<int, 2>{}, c);
      }
      cluster_sync_all();                                      // nobody leaves while its partials are being read
    }
  } else if (split > 1) {
    cluster_sync_all();
    cluster_sync_all();
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tc_dealloc(tmem, tmem_cols(MT));
  }
}

bool encode_bf16_rows(CUtensorMap* map, const void* base, uint64_t inner, uint64_t rows, uint64_t stride_elems, uint32_t box_rows) {
  EncodeTiledFn fn = tensor_map_encoder();
  if (!fn) return false;
  const cuuint64_t dims[2] = {inner, rows};
  const cuuint64_t strides[1] = {stride_elems * 2};
  const cuuint32_t box[2] = {kBlockK, box_rows};
  const cuuint32_t elem_strides[2] = {1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem_strides,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int EPI, int MT, bool GROUPED>
int launch(const cacheir_b200_dense_args& p, int split, cudaStream_t stream, const Groups& groups) {
  constexpr size_t kSmem = 1024 + static_cast<size_t>(num_stages(MT)) * stage_bytes(MT) + kTailBytes;
  static_assert(kSmem * ctas_per_sm(MT) <= 227 * 1024, "ring must fit");
  static_assert(static_cast<size_t>(MT) * kTileN * 4 <= static_cast<size_t>(num_stages(MT)) * stage_bytes(MT), "partials must fit the ring");
  CUtensorMap tw, tx;
  const uint64_t w_rows = p.batch > 1 ? static_cast<uint64_t>(p.w_batch_rows) * (p.batch - 1) + p.N : p.N;
  const uint64_t x_cols = GROUPED ? p.K : static_cast<uint64_t>(p.x_batch_cols) * (p.batch - 1) + p.K;
  if (!encode_bf16_rows(&tw, p.w, p.K, w_rows, p.w_stride, kTileN) ||
      !encode_bf16_rows(&tx, p.x, x_cols, GROUPED ? groups.x_rows : p.T, p.x_stride, MT))
    return CACHEIR_B200_EUNSUPPORTED;
  auto kern = dense_gemm_kernel<EPI, MT, GROUPED>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kSmem));
  if (e != cudaSuccess) return static_cast<int>(e);
  const int n_tiles = (p.N + kTileN - 1) / kTileN;
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = GROUPED ? dim3((groups.place_of ? 0 : p.T / MT) + (p.T < p.batch ? p.T : p.batch), split, n_tiles) : dim3((p.T + MT - 1) / MT, split, n_tiles * p.batch);
  cfg.blockDim = dim3(kThreads, 1, 1);
  cfg.dynamicSmemBytes = kSmem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = split;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = split > 1 ? 1 : 0;
  e = cudaLaunchKernelEx(&cfg, kern, tw, tx, p, n_tiles, groups);
  if (e != cudaSuccess) return static_cast<int>(e);
  return launch_status();
}

}  // namespace
}  // namespace cb200
