// Talking-heads attention over a paged cache, sm_100a: preparation, the plain form, and decoding.
//
// prepare   rotation, value norm, the new cache rows; queries as they are or mixed. Mixing scores is linear, so head h's mixed score
//           is one product of a whole cached key row with a query that holds, per key/value head, sum_g talk[h, g] q_g.
// simple    any extents, float32 arithmetic: one CTA per row, all heads.
// step      one CTA per (sequence, split, set of key/value heads). Tiles of 16 or 32 cached tokens land in a ring as TMA boxes of 64
//           columns. Eight warps with warp MMAs: raw scores of all heads (up to 16 heads of a key/value head, a band, being the 16-row
//           operand) go to shared memory as sums of two bf16 numbers; then a band's warp has its mixed scores as one more product,
//           its softmax and its values in registers. One barrier per tile. Splits meet in distributed shared memory. Sets read all
//           keys and their own values; there is one unless the output would not fit the registers.
#include "talking_attention.cuh"

namespace cb200 {
namespace {

using Args = cacheir_b200_talking_args;

__device__ int g_talking_status = 0;

struct PrepareParams {
  Args a;
  long long q_stride, k_stride, v_stride;
  const float2* table;
  int table_positions, rot_dims;
  float eps;
};

// Entry c of a head's row as rotated by the angles of one position.
template <typename T>
__device__ __forceinline__ float rotated(const T* src, int c, int half, const float2* cs) {
  const float x = Elem<T>::ld(src + c);
  if (c >= 2 * half) return x;
  const bool low = c < half;
  const float other = Elem<T>::ld(src + (low ? c + half : c - half));
  const float2 t = cs[low ? c : c - half];
  return low ? x * t.x - other * t.y : x * t.x + other * t.y;
}

// A warp per head: queries, keys, values. MIXED (heads of a key/value head, padded; more than kHeldHeads: any number): one block has
// a row, and its queries go through shared memory.
constexpr int kHeldHeads = 8;
template <typename T, int MIXED>
__global__ void __launch_bounds__(256)
talking_prepare_kernel(const PrepareParams p, const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, T* __restrict__ q_out) {
  extern __shared__ float sm[];                  // MIXED: [heads][dim] queries, [heads][heads] talk
  const Args& a = p.a;
  const int row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int seg = a.row_seg[row], pos = a.positions[row];
  if (seg < 0 || pos < 0 || pos >= p.table_positions || pos / a.page_size >= a.max_pages) return;
  const int slot = a.page_table[static_cast<size_t>(seg) * a.max_pages + pos / a.page_size];
  const bool cached = slot >= 0 && slot < a.num_slots;
  const size_t at = static_cast<size_t>(max(slot, 0)) * a.page_size + pos % a.page_size;
  const int half = p.rot_dims / 2, units = a.heads + 2 * a.kv_heads;
  const float2* cs = p.table + static_cast<size_t>(pos) * half;
  for (int u = blockIdx.y * 8 + warp; u < units; u += gridDim.y * 8) {
    if (u < a.heads) {
      const T* src = q + static_cast<size_t>(row) * p.q_stride + static_cast<size_t>(u) * a.dim;
      for (int c = lane; c < a.dim; c += 32) {
        const float x = rotated(src, c, half, cs);
        if (MIXED > 0) sm[u * a.dim + c] = a.scale < 0.f ? -x : x;
        else Elem<T>::st(q_out + (static_cast<size_t>(row) * a.heads + u) * a.dim + c, x);
      }
    } else if (!cached) {
      continue;
    } else if (u < a.heads + a.kv_heads) {
      const int g = u - a.heads;
      const T* src = k + static_cast<size_t>(row) * p.k_stride + static_cast<size_t>(g) * a.dim;
      T* dst = static_cast<T*>(a.keys) + (at * a.kv_heads + g) * a.dim;
      for (int c = lane; c < a.dim; c += 32) Elem<T>::st(dst + c, rotated(src, c, half, cs));
    } else {
      const int g = u - a.heads - a.kv_heads;
      const T* src = v + static_cast<size_t>(row) * p.v_stride + static_cast<size_t>(g) * a.vdim;
      T* dst = static_cast<T*>(a.values) + (at * a.kv_heads + g) * a.vdim;
      float ss = 0.f;
      for (int c = lane; c < a.vdim; c += 32) {
        const float x = Elem<T>::ld(src + c);
        ss = fmaf(x, x, ss);
      }
      const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(a.vdim) + p.eps);
      for (int c = lane; c < a.vdim; c += 32) Elem<T>::st(dst + c, Elem<T>::ld(src + c) * inv);
    }
  }
  if constexpr (MIXED > 0) {
    float* s_talk = sm + a.heads * a.dim;
    for (int i = threadIdx.x; i < a.heads * a.heads; i += 256) s_talk[i] = a.talk[i];
    __syncthreads();
    // a thread has eight columns of a key row and some of the heads that meet them
    const int group = a.heads / a.kv_heads, width = a.kv_heads * a.dim, pieces = width / 8;
    const int shares = pieces >= 256 ? 1 : min(256 / pieces, a.heads);
    for (int u = threadIdx.x; u < pieces * shares; u += 256) {
      const int c = u % pieces * 8, share = u / pieces, g = c / a.dim, d = c % a.dim;
      const float* src = sm + g * group * a.dim + d;
      const float* talk = s_talk + g * group;
      T* dst = q_out + static_cast<size_t>(row) * a.heads * width + c;
      auto leave = [&](int h, const float (&y)[8]) {
        if constexpr (sizeof(T) == 2) {
          VecIO<T, 8>::st(dst + static_cast<size_t>(h) * width, y);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) Elem<T>::st(dst + static_cast<size_t>(h) * width + e, y[e]);
        }
      };
      if constexpr (MIXED <= kHeldHeads) {
        float x[MIXED][8];
#pragma unroll
        for (int i = 0; i < MIXED; ++i)
#pragma unroll
          for (int e = 0; e < 8; ++e) x[i][e] = i < group ? src[i * a.dim + e] : 0.f;
        for (int h = share; h < a.heads; h += shares) {
          float y[8] = {};
#pragma unroll
          for (int i = 0; i < MIXED; ++i) {
            const float t = i < group ? talk[h * a.heads + i] : 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] = fmaf(t, x[i][e], y[e]);
          }
          leave(h, y);
        }
      } else {
        for (int h = share; h < a.heads; h += shares) {
          float y[8] = {};
          for (int i = 0; i < group; ++i) {
            const float t = talk[h * a.heads + i];
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] = fmaf(t, src[i * a.dim + e], y[e]);
          }
          leave(h, y);
        }
      }
    }
  }
}

// ---- plain form ------------------------------------------------------------------------------------------------------
constexpr int kSimpleKeys = 32;
template <typename T>
__global__ void __launch_bounds__(256)
talking_simple_kernel(const Args a, const T* __restrict__ q, T* __restrict__ out) {
  extern __shared__ float sm[];
  float* s_q = sm;                               // [heads][dim]
  float* s_o = s_q + a.heads * a.dim;            // [heads][vdim]
  float* s_raw = s_o + a.heads * a.vdim;         // [heads][keys]
  float* s_p = s_raw + a.heads * kSimpleKeys;    // [heads][keys]
  float* s_m = s_p + a.heads * kSimpleKeys;      // [heads] reference, sum, factor of what came before
  float* s_l = s_m + a.heads;
  float* s_f = s_l + a.heads;
  const int row = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seg = a.row_seg[row];
  if (seg < 0) return;
  const int pos = a.positions[row], group = a.heads / a.kv_heads;
  for (int c = tid; c < a.heads * a.dim; c += 256) s_q[c] = Elem<T>::ld(q + static_cast<size_t>(row) * a.heads * a.dim + c);
  for (int c = tid; c < a.heads * a.vdim; c += 256) s_o[c] = 0.f;
  for (int h = tid; h < a.heads; h += 256) { s_m[h] = 0.f; s_l[h] = 1.f; }      // the score 0 that has no value
  auto cached = [&](int j) { return static_cast<size_t>(talk_slot(a, seg, j / a.page_size)) * a.page_size + j % a.page_size; };
  for (int k0 = max(0, pos - a.window + 1); k0 <= pos; k0 += kSimpleKeys) {
    const int n = min(kSimpleKeys, pos + 1 - k0);
    __syncthreads();
    for (int i = tid; i < a.heads * kSimpleKeys; i += 256) {
      const int h = i / kSimpleKeys, j = i % kSimpleKeys;
      float dot = 0.f;
      if (j < n) {
        const T* key = static_cast<const T*>(a.keys) + (cached(k0 + j) * a.kv_heads + h / group) * a.dim;
        for (int c = 0; c < a.dim; ++c) dot = fmaf(s_q[h * a.dim + c], Elem<T>::ld(key + c), dot);
      }
      s_raw[i] = dot * a.scale;
    }
    __syncthreads();
    for (int h = warp; h < a.heads; h += 8) {
      float s = 0.f;
      for (int g = 0; g < a.heads; ++g) s = fmaf(a.talk[static_cast<size_t>(h) * a.heads + g], s_raw[g * kSimpleKeys + lane], s);
      if (lane >= n) s = -INFINITY;
      const float before = s_m[h], top = fmaxf(before, warp_max(s));
      const float e = lane < n ? expf(s - top) : 0.f, sum = warp_sum(e);
      s_p[h * kSimpleKeys + lane] = e;
      __syncwarp();
      if (lane == 0) {
        const float f = expf(before - top);
        s_f[h] = f;
        s_m[h] = top;
        s_l[h] = s_l[h] * f + sum;
      }
    }
    __syncthreads();
    for (int i = tid; i < a.heads * a.vdim; i += 256) {
      const int h = i / a.vdim, c = i % a.vdim;
      float acc = s_o[i] * s_f[h];
      for (int j = 0; j < n; ++j)
        acc = fmaf(s_p[h * kSimpleKeys + j], Elem<T>::ld(static_cast<const T*>(a.values) + (cached(k0 + j) * a.kv_heads + h / group) * a.vdim + c), acc);
      s_o[i] = acc;
    }
  }
  __syncthreads();
  for (int i = tid; i < a.heads * a.vdim; i += 256)
    Elem<T>::st(out + static_cast<size_t>(row) * a.heads * a.vdim + i, s_o[i] / s_l[i / a.vdim]);
}

// ---- decoding --------------------------------------------------------------------------------------------------------
constexpr int kWarps = 8;                        // consumer warps; one more copies
constexpr int kConsumers = kWarps * 32;
constexpr int kStepThreads = kConsumers + 32;
constexpr int kMaxStages = 6;
constexpr int kMaxSplits = 8;                    // CTAs of a cluster
constexpr int kMaxTiles = 16;                    // 16 x 16 output tiles per warp

struct StepShape {
  int sets, tile, stages;                        // sets of key/value heads, cached tokens per tile
  int k_boxes, v_boxes;
  int bands;                                     // of a set at most: a band is up to 16 heads of one key/value head
  int shares;                                    // warps that share a band's value columns
  int bands_per_warp, pairs_per_warp;            // pairs of 8-column tiles
  size_t ring, smem;
};
struct StepParams {
  Args a;
  const __nv_bfloat16* q;
  __nv_bfloat16* out;
  StepShape s;
  int splits;
};

__host__ __device__ inline int round_to(int n, int m) { return (n + m - 1) / m * m; }
// Parts behind the ring, in bytes: barriers; talk [bands][16][heads], scores [2][hi, lo][heads][tile], queries [heads][dim] as bf16
// with rows 16 bytes over a multiple of 16 entries; reference and sum of a set's heads.
struct StepSpace {
  int talk_pitch, score_pitch, q_pitch, talk, scores, q, meet, total;
  __host__ __device__ StepSpace(int heads, int dim, int bands, int set_heads, int tile) {
    const int h16 = round_to(heads, 16);
    talk_pitch = h16 + 8;
    score_pitch = tile + 8;
    q_pitch = round_to(dim, 16) + 8;
    talk = 2 * kMaxStages * 8;
    scores = talk + bands * 16 * talk_pitch * 2;
    q = scores + 4 * h16 * score_pitch * 2;
    meet = q + heads * q_pitch * 2;
    total = meet + 2 * round_to(set_heads, 4) * 4;
  }
};

__device__ __forceinline__ float ld_peer_f32(const float* local, uint32_t rank) {
  uint32_t remote;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(smem_addr(local)), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
  return v;
}
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ void consumers_sync() { asm volatile("barrier.cta.sync 1, %0;" ::"n"(kConsumers) : "memory"); }

// BANDS, PAIRS: what a warp has of the output at most
template <int BANDS, int PAIRS, int TILE>
__global__ void __launch_bounds__(kStepThreads, 1)
talking_step_kernel(const __grid_constant__ CUtensorMap tmap_k, const __grid_constant__ CUtensorMap tmap_v, const StepParams p) {
  constexpr int kBox = TILE * 128, kBlocks = TILE / 16;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const Args& a = p.a;
  const int group = a.heads / a.kv_heads, subs = (group + 15) / 16;
  const int split = blockIdx.x, seg = blockIdx.z;          // (the cluster spans the whole x extent)
  const int kv0 = a.kv_heads * static_cast<int>(blockIdx.y) / p.s.sets, kv1 = a.kv_heads * (static_cast<int>(blockIdx.y) + 1) / p.s.sets;
  const int head0 = kv0 * group, set_heads = (kv1 - kv0) * group, bands = (kv1 - kv0) * subs, h16 = round_to(a.heads, 16);
  const int stage_bytes = (p.s.k_boxes + p.s.v_boxes) * kBox;
  const StepSpace space(a.heads, a.dim, p.s.bands, p.s.bands / subs * group, TILE);
  uint8_t* rest = smem + p.s.ring;
  uint64_t* full = reinterpret_cast<uint64_t*>(rest);
  uint64_t* empty = full + kMaxStages;
  __nv_bfloat16* s_talk = reinterpret_cast<__nv_bfloat16*>(rest + space.talk);
  __nv_bfloat16* s_score = reinterpret_cast<__nv_bfloat16*>(rest + space.scores);
  __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(rest + space.q);
  float* s_m = reinterpret_cast<float*>(rest + space.meet);
  float* s_l = s_m + round_to(p.s.bands / subs * group, 4);
  const int plane = h16 * space.score_pitch;               // of s_score: [buffer][hi, lo]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (a.row_seg[seg] < 0) return;                          // (a padding row: the whole cluster leaves)
  const int pos = a.positions[seg];
  const int tile_lo = max(0, pos - a.window + 1) / TILE, tiles = pos / TILE - tile_lo + 1;
  const int begin = tiles * split / p.splits, n = tiles * (split + 1) / p.splits - begin;

  if (threadIdx.x == 0) {
    for (int s = 0; s < p.s.stages; ++s) { ptx::mbar_init(smem_addr(&full[s]), 1); ptx::mbar_init(smem_addr(&empty[s]), kWarps); }
    ptx::mbar_fence_init();
  }
  __syncthreads();

  const int g4 = lane >> 2, t4 = lane & 3, lrow = lane & 7, lmat = lane >> 3;
  const int pairs = (a.vdim + 15) / 16, share = warp % p.s.shares, band0 = warp / p.s.shares;
  float o[BANDS][PAIRS][2][4], m_run[BANDS][2], l_run[BANDS][2];
#pragma unroll
  for (int i = 0; i < BANDS; ++i) {
    m_run[i][0] = m_run[i][1] = -1e30f;
    l_run[i][0] = l_run[i][1] = 0.f;
#pragma unroll
    for (int j = 0; j < PAIRS; ++j)
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][j][t][e] = 0.f;
  }

  if (warp == kWarps) {
    // ---------------- copies: a lane per box ----------------
    const int boxes = p.s.k_boxes + p.s.v_boxes;
    int issued = 0;
    bool ok = true;
    for (int it = 0; it < n && ok; ++it) {
      const int s = it % p.s.stages, key0 = (tile_lo + begin + it) * TILE;
      if (it >= p.s.stages) ok = ptx::mbar_wait(smem_addr(&empty[s]), ((it / p.s.stages) & 1) ^ 1, &g_talking_status, (10 << 8) | 1);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const uint32_t bar = smem_addr(&full[s]), dst = smem_addr(smem + s * stage_bytes);
      const int row = talk_slot(a, seg, key0 / kTalkPage) * kTalkPage + key0 % kTalkPage;
      if (lane == 0) ptx::mbar_expect_tx(bar, stage_bytes);
      __syncwarp();
      for (int b = lane; b < boxes; b += 32) {
        if (b < p.s.k_boxes) ptx::tma_load_2d(dst + b * kBox, &tmap_k, bar, b * 64, row);
        else ptx::tma_load_2d(dst + b * kBox, &tmap_v, bar, kv0 * a.vdim + (b - p.s.k_boxes) * 64, row);
      }
      issued = it + 1;
    }
    if (issued < n)                      // a wait gave up: nothing may still be on its way when the block ends
      for (int it = max(0, issued - p.s.stages); it < issued; ++it)
        ptx::mbar_wait(smem_addr(&full[it % p.s.stages]), (it / p.s.stages) & 1, &g_talking_status, (10 << 8) | 2);
    __syncwarp();
  } else {
    // queries and talk, while the first tiles travel
    for (int h = warp; h < a.heads; h += kWarps)
      for (int c = lane; c < space.q_pitch; c += 32)
        s_q[h * space.q_pitch + c] = c < a.dim ? p.q[(static_cast<size_t>(seg) * a.heads + h) * a.dim + c] : __float2bfloat16_rn(0.f);
    for (int r = warp; r < bands * 16; r += kWarps) {
      const int h = (r >> 4) % subs * 16 + (r & 15), head = head0 + (r >> 4) / subs * group + h;
      for (int g = lane; g < h16; g += 32)
        s_talk[r * space.talk_pitch + g] = __float2bfloat16_rn(h < group && g < a.heads ? a.talk[static_cast<size_t>(head) * a.heads + g] : 0.f);
    }
    for (int i = threadIdx.x; i < 4 * plane; i += kConsumers) s_score[i] = __float2bfloat16_rn(0.f);      // (rows behind the last head stay zero)
    consumers_sync();

    for (int it = 0; it < n; ++it) {
      const int s = it % p.s.stages, key0 = (tile_lo + begin + it) * TILE;
      // (a wait that gave up is on record; everyone goes on, so that the barriers below still meet)
      ptx::mbar_wait(smem_addr(&full[s]), (it / p.s.stages) & 1, &g_talking_status, (10 << 8) | 3);
      __syncwarp();
      uint8_t* k_tile = smem + s * stage_bytes;
      uint8_t* v_tile = k_tile + p.s.k_boxes * kBox;
      const uint32_t k_at = smem_addr(k_tile), v_at = smem_addr(v_tile);
      __nv_bfloat16* score = s_score + (it & 1) * 2 * plane;
      // values behind the last token may be anything: zero, so that 0 * value stays 0
      if (key0 + TILE - 1 > pos) {
        const int valid = pos + 1 - key0;
        for (int i = threadIdx.x; i < (TILE - valid) * p.s.v_boxes * 8; i += kConsumers) {
          const int r = valid + i / (p.s.v_boxes * 8), c = i % (p.s.v_boxes * 8);
          *reinterpret_cast<uint4*>(v_tile + (c >> 3) * kBox + r * 128 + (c & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
      }
      // raw scores of all heads: a band and 16 keys at a time
      for (int u = warp; u < a.kv_heads * subs * kBlocks; u += kWarps) {
        const int kb = u % kBlocks, band = u / kBlocks, g = subs == 1 ? band : band / subs, sub = subs == 1 ? 0 : band % subs;
        const int h0 = g * group + sub * 16, count = min(16, group - sub * 16);
        float sc[2][4], sd[2][4];        // even and odd steps in sums of their own (shorter dependent chains)
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int e = 0; e < 4; ++e) sc[t][e] = sd[t][e] = 0.f;
        const uint32_t qa = smem_addr(s_q) + (min(h0 + (lane & 15), a.heads - 1) * space.q_pitch + (lane >> 4) * 8) * 2;
        const int key = kb * 16 + (lmat >> 1) * 8 + lrow, last_piece = p.s.k_boxes * 8 - 1, piece0 = g * a.dim / 8 + (lmat & 1);
        const uint32_t row_at = k_at + key * 128;
        auto step = [&](int k, float (&x)[2][4]) {
          uint32_t af[4], bf[4];
          ldsm_x4(qa + k * 32, af);
          const int c = min(piece0 + 2 * k, last_piece);      // (a piece behind the head meets zero queries)
          ldsm_x4(row_at + (c >> 3) * kBox + (((c & 7) ^ lrow) << 4), bf);
          mma_bf16(x[0], af, bf[0], bf[1]);
          mma_bf16(x[1], af, bf[2], bf[3]);
        };
        const int steps = (a.dim + 15) / 16;
        int k = 0;
#pragma unroll 2
        for (; k + 1 < steps; k += 2) { step(k, sc); step(k + 1, sd); }
        if (k < steps) step(k, sc);
#pragma unroll
        for (int r = 0; r < 2; ++r)
          if (g4 + r * 8 < count)
#pragma unroll
            for (int t = 0; t < 2; ++t) {
              const float x = (sc[t][2 * r] + sd[t][2 * r]) * a.scale, y = (sc[t][2 * r + 1] + sd[t][2 * r + 1]) * a.scale;
              float xh, xl, yh, yl;
              split_bf16(x, &xh, &xl);
              split_bf16(y, &yh, &yl);
              __nv_bfloat16* dst = score + (h0 + g4 + r * 8) * space.score_pitch + kb * 16 + t * 8 + 2 * t4;
              *reinterpret_cast<uint32_t*>(dst) = pack_bf16(xh, yh);
              *reinterpret_cast<uint32_t*>(dst + plane) = pack_bf16(xl, yl);
            }
      }
      consumers_sync();
#pragma unroll
      for (int i = 0; i < BANDS; ++i) {
        const int band = band0 + i * kWarps;
        if (band >= bands) break;
        // the band's mixed scores: talk (exact in bf16) times both halves of the raw ones
        float x[kBlocks][2][4];
#pragma unroll
        for (int kb = 0; kb < kBlocks; ++kb)
#pragma unroll
          for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) x[kb][t][e] = 0.f;
        const uint32_t ta = smem_addr(s_talk) + ((band * 16 + (lane & 15)) * space.talk_pitch + (lane >> 4) * 8) * 2;
        const uint32_t sa = smem_addr(score) + (((lmat & 1) * 8 + lrow) * space.score_pitch + (lmat >> 1) * 8) * 2;
#pragma unroll 2
        for (int k = 0; k < h16; k += 16) {
          uint32_t af[4];
          ldsm_x4(ta + k * 2, af);
#pragma unroll
          for (int kb = 0; kb < kBlocks; ++kb)
#pragma unroll
            for (int part = 0; part < 2; ++part) {
              uint32_t bf[4];
              ldsm_x4_t(sa + (part * plane + k * space.score_pitch + kb * 16) * 2, bf);
              mma_bf16(x[kb][0], af, bf[0], bf[1]);
              mma_bf16(x[kb][1], af, bf[2], bf[3]);
            }
        }
        const int base = key0 + 2 * t4;
        float top[2] = {m_run[i][0], m_run[i][1]}, corr[2];
#pragma unroll
        for (int kb = 0; kb < kBlocks; ++kb)
#pragma unroll
          for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int key = base + kb * 16 + t * 8 + (e & 1);
              x[kb][t][e] = key <= pos && key > pos - a.window ? x[kb][t][e] * kTalkLog2e : -INFINITY;
              top[e >> 1] = fmaxf(top[e >> 1], x[kb][t][e]);
            }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 1));
          top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 2));
          corr[r] = talk_ex2(m_run[i][r] - top[r]);
          m_run[i][r] = top[r];
          l_run[i][r] *= corr[r];
        }
        uint32_t pa[kBlocks][4];
#pragma unroll
        for (int kb = 0; kb < kBlocks; ++kb)
#pragma unroll
          for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
              const float u = talk_ex2(x[kb][t][2 * r] - top[r]), v = talk_ex2(x[kb][t][2 * r + 1] - top[r]);
              l_run[i][r] += u + v;
              pa[kb][t * 2 + r] = pack_bf16(u, v);
            }
        if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
          for (int j = 0; j < PAIRS; ++j)
#pragma unroll
            for (int t = 0; t < 2; ++t) { o[i][j][t][0] *= corr[0]; o[i][j][t][1] *= corr[0]; o[i][j][t][2] *= corr[1]; o[i][j][t][3] *= corr[1]; }
        }
        const int piece0 = (subs == 1 ? band : band / subs) * a.vdim / 8 + (lmat >> 1), last_piece = p.s.v_boxes * 8 - 1;
        const uint32_t row_at = v_at + ((lmat & 1) * 8 + lrow) * 128;
#pragma unroll
        for (int j = 0; j < PAIRS; ++j) {
          const int pair = share + j * p.s.shares;
          if (pair < pairs) {
            const int c = min(piece0 + 2 * pair, last_piece);      // (columns behind the head are not kept)
            const uint32_t at = row_at + (c >> 3) * kBox + (((c & 7) ^ lrow) << 4);
#pragma unroll
            for (int kb = 0; kb < kBlocks; ++kb) {
              uint32_t bf[4];
              ldsm_x4_t(at + kb * 16 * 128, bf);
              mma_bf16(o[i][j][0], pa[kb], bf[0], bf[1]);
              mma_bf16(o[i][j][1], pa[kb], bf[2], bf[3]);
            }
          }
        }
      }
      __syncwarp();
      if (lane == 0) ptx::mbar_arrive(smem_addr(&empty[s]));
    }
  }

  // ---------------- outputs over the drained ring, then the cluster's CTAs meet ----------------
  __syncthreads();
  float* s_o = reinterpret_cast<float*>(smem);                  // [set_heads][vdim]
  if (warp < kWarps) {
#pragma unroll
    for (int i = 0; i < BANDS; ++i) {
      const int band = band0 + i * kWarps;
      if (band >= bands) break;
      const int sub = band % subs, h0 = band / subs * group + sub * 16, count = min(16, group - sub * 16);
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        l_run[i][r] += __shfl_xor_sync(0xffffffffu, l_run[i][r], 1);
        l_run[i][r] += __shfl_xor_sync(0xffffffffu, l_run[i][r], 2);
        if (share == 0 && t4 == 0 && g4 + r * 8 < count) {
          s_m[h0 + g4 + r * 8] = m_run[i][r];
          s_l[h0 + g4 + r * 8] = l_run[i][r];
        }
      }
#pragma unroll
      for (int j = 0; j < PAIRS; ++j)
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int r = g4 + (e >> 1) * 8, c = (share + j * p.s.shares) * 16 + t * 8 + 2 * t4 + (e & 1);
            if (r < count && c < a.vdim) s_o[(h0 + r) * a.vdim + c] = o[i][j][t][e];
          }
    }
  }
  __syncthreads();
  auto finish = [&](int i, float m, float l, float acc) {       // the score 0 without a value joins here
    const float top = fmaxf(m, 0.f), by = talk_ex2(m - top);
    const float y = acc * by / (l * by + talk_ex2(-top));
    p.out[(static_cast<size_t>(seg) * a.heads + head0) * a.vdim + i] = __float2bfloat16_rn(y);
  };
  const int total = set_heads * a.vdim;
  if (p.splits == 1) {
    for (int i = threadIdx.x; i < total; i += kStepThreads) finish(i, s_m[i / a.vdim], s_l[i / a.vdim], s_o[i]);
    return;
  }
  __syncwarp();
  cluster_sync_all();
  for (int i = split * kStepThreads + threadIdx.x; i < total; i += p.splits * kStepThreads) {
    const int h = i / a.vdim;
    float ms[kMaxSplits], m = -1e30f, l = 0.f, acc = 0.f;
#pragma unroll
    for (int r = 0; r < kMaxSplits; ++r) {
      ms[r] = r < p.splits ? ld_peer_f32(s_m + h, r) : -1e30f;
      m = fmaxf(m, ms[r]);
    }
#pragma unroll
    for (int r = 0; r < kMaxSplits; ++r)
      if (r < p.splits) {
        const float by = talk_ex2(ms[r] - m);
        l = fmaf(ld_peer_f32(s_l + h, r), by, l);
        acc = fmaf(ld_peer_f32(s_o + i, r), by, acc);
      }
    finish(i, m, l, acc);
  }
  __syncwarp();
  cluster_sync_all();                      // nobody leaves while its part is being read
}

constexpr size_t kSmemLimit = 227 * 1024;
// Everything a launch needs to know about its shared memory; stages == 0: these extents do not fit.
StepShape step_shape(int heads, int kv_heads, int dim, int vdim) {
  StepShape s{};
  const int group = heads / kv_heads, subs = (group + 15) / 16, pairs = (vdim + 15) / 16;
  for (int sets = 1; sets <= kv_heads; ++sets) {
    const int kv_per_set = (kv_heads + sets - 1) / sets;
    s.sets = sets;
    s.bands = kv_per_set * subs;
    s.shares = s.bands < kWarps ? kWarps / s.bands : 1;
    s.bands_per_warp = (s.bands + kWarps - 1) / kWarps;
    s.pairs_per_warp = (pairs + s.shares - 1) / s.shares;
    if (s.bands_per_warp > 2 || s.bands_per_warp * s.pairs_per_warp > kMaxTiles) continue;
    s.k_boxes = (kv_heads * dim + 63) / 64;
    s.v_boxes = (kv_per_set * vdim + 63) / 64;
    for (int tile : {32, 16}) {
      s.tile = tile;
      const size_t rest = 1024 + StepSpace(heads, dim, s.bands, kv_per_set * group, tile).total;
      const size_t stage = static_cast<size_t>(s.k_boxes + s.v_boxes) * tile * 128;
      if (rest + 2 * stage > kSmemLimit) continue;
      size_t stages = (kSmemLimit - rest) / stage;
      if (stages > kMaxStages) stages = kMaxStages;
      if (tile == 32 && stages < 3) continue;
      if (static_cast<size_t>(kv_per_set) * group * vdim * 4 > stages * stage) continue;      // the outputs meet in the ring
      s.stages = static_cast<int>(stages);
      s.ring = stages * stage;
      s.smem = rest + s.ring;
      return s;
    }
  }
  s.stages = 0;
  return s;
}

template <int BANDS, int PAIRS, int TILE>
int launch_step(const StepParams& p, cudaStream_t st) {
  const Args& a = p.a;
  CUtensorMap tk, tv;
  const uint64_t rows = static_cast<uint64_t>(a.num_slots) * kTalkPage;
  if (!talk_encode(&tk, a.keys, static_cast<uint64_t>(a.kv_heads) * a.dim, rows, TILE) ||
      !talk_encode(&tv, a.values, static_cast<uint64_t>(a.kv_heads) * a.vdim, rows, TILE))
    return CACHEIR_B200_EUNSUPPORTED;
  auto kern = talking_step_kernel<BANDS, PAIRS, TILE>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(p.s.smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(p.splits, p.s.sets, a.rows);
  cfg.blockDim = dim3(kStepThreads, 1, 1);
  cfg.dynamicSmemBytes = p.s.smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = p.splits;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = p.splits > 1 ? 1 : 0;
  e = cudaLaunchKernelEx(&cfg, kern, tk, tv, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  return launch_status();
}

template <int BANDS, int PAIRS>
int launch_tile(const StepParams& p, cudaStream_t st) {
  return p.s.tile == 32 ? launch_step<BANDS, PAIRS, 32>(p, st) : launch_step<BANDS, PAIRS, 16>(p, st);
}

}  // namespace
}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_talking_prepare(const cacheir_b200_talking_args* args, const void* q, long long q_stride, const void* k,
                                            long long k_stride, const void* v, long long v_stride, int rot_dims, const float* rope_table,
                                            int rope_positions, float eps, int mixed, void* q_out, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_talking_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!talk_args_ok(a) || !q || !k || !v || !q_out || rot_dims < 0 || rot_dims % 2 != 0 || rot_dims > a.dim || (rot_dims > 0 && !rope_table) ||
      rope_positions <= 0)
    return CACHEIR_B200_EINVAL;
  const PrepareParams p{a, q_stride, k_stride, v_stride, reinterpret_cast<const float2*>(rope_table), rope_positions, rot_dims, eps};
  const int group = a.heads / a.kv_heads;
  cudaStream_t st = as_stream(stream);
  if (!mixed) {
    const dim3 grid(a.rows, (a.heads + 2 * a.kv_heads + 7) / 8);
    if (grid.y > 65535) return CACHEIR_B200_ELIMIT;
    CB200_HYBRID_DTYPE(a.dtype, (talking_prepare_kernel<T, 0><<<grid, 256, 0, st>>>(p, static_cast<const T*>(q), static_cast<const T*>(k),
                                                                                     static_cast<const T*>(v), static_cast<T*>(q_out))));
    return launch_status();
  }
  if (a.dim % 8 != 0 || !aligned_to(q_out, 16)) return CACHEIR_B200_EUNSUPPORTED;
  const size_t smem = (static_cast<size_t>(a.heads) * a.dim + static_cast<size_t>(a.heads) * a.heads) * 4;
  if (smem > 200 * 1024) return CACHEIR_B200_ELIMIT;
#define CB200_MIX(MIXED)                                                                                                              \
  {                                                                                                                                   \
    const cudaError_t e = cudaFuncSetAttribute(talking_prepare_kernel<T, MIXED>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)); \
    if (e != cudaSuccess) return static_cast<int>(e);                                                                                 \
    talking_prepare_kernel<T, MIXED><<<dim3(a.rows, 1), 256, smem, st>>>(p, static_cast<const T*>(q), static_cast<const T*>(k),        \
                                                                         static_cast<const T*>(v), static_cast<T*>(q_out));           \
  }
  CB200_HYBRID_DTYPE(a.dtype, {
    if (group == 1) CB200_MIX(1)
    else if (group == 2) CB200_MIX(2)
    else if (group <= 4) CB200_MIX(4)
    else if (group <= kHeldHeads) CB200_MIX(kHeldHeads)
    else CB200_MIX(kHeldHeads + 1)
  });
#undef CB200_MIX
  return launch_status();
}

extern "C" int cacheir_b200_talking_simple(const cacheir_b200_talking_args* args, const void* q, void* out, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_talking_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!talk_args_ok(a) || !q || !out) return CACHEIR_B200_EINVAL;
  const size_t smem = static_cast<size_t>(a.heads) * (a.dim + a.vdim + 2 * kSimpleKeys + 3) * 4;
  if (smem > kSmemLimit) return CACHEIR_B200_ELIMIT;
  CB200_HYBRID_DTYPE(a.dtype, {
    const cudaError_t e = cudaFuncSetAttribute(talking_simple_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    talking_simple_kernel<T><<<a.rows, 256, smem, as_stream(stream)>>>(a, static_cast<const T*>(q), static_cast<T*>(out));
  });
  return launch_status();
}

extern "C" int cacheir_b200_talking_step_supported(int heads, int kv_heads, int dim, int vdim, int page_size, int dtype) {
  return dtype == CACHEIR_B200_BF16 && page_size == kTalkPage && kv_heads > 0 && heads % kv_heads == 0 && dim >= 8 && dim % 8 == 0 && vdim >= 8 &&
         vdim % 8 == 0 && step_shape(heads, kv_heads, dim, vdim).stages > 0 ? 1 : 0;
}

extern "C" int cacheir_b200_talking_step_splits(int rows, int heads, int kv_heads, int dim, int vdim, int window, int max_pages, int page_size) {
  if (rows <= 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || page_size <= 0) return 1;
  const StepShape shape = step_shape(heads, kv_heads, dim, vdim);
  long long pages = (static_cast<long long>(window) + page_size - 2) / page_size + 1;
  if (pages > max_pages) pages = max_pages;
  long long s = kNumSMs / (static_cast<long long>(rows) * shape.sets);
  if (s > pages) s = pages;              // at least a page each
  return s < 1 ? 1 : static_cast<int>(s > kMaxSplits ? kMaxSplits : s);
}

extern "C" int cacheir_b200_talking_step(const cacheir_b200_talking_args* args, const void* q, void* out, int splits, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_talking_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!talk_args_ok(a) || !q || !out || !a.decode || a.rows != a.segments) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_talking_step_supported(a.heads, a.kv_heads, a.dim, a.vdim, a.page_size, a.dtype)) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(a.keys, 16) || !aligned_to(a.values, 16)) return CACHEIR_B200_EALIGN;
  if (splits <= 0) splits = cacheir_b200_talking_step_splits(a.rows, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.max_pages, a.page_size);
  if (splits > kMaxSplits || a.rows > 65535) return CACHEIR_B200_ELIMIT;
  const StepParams p{a, static_cast<const __nv_bfloat16*>(q), static_cast<__nv_bfloat16*>(out), step_shape(a.heads, a.kv_heads, a.dim, a.vdim), splits};
  cudaStream_t st = as_stream(stream);
  const int pairs = p.s.pairs_per_warp;
  if (p.s.bands_per_warp == 2) return pairs <= 4 ? launch_tile<2, 4>(p, st) : launch_tile<2, 8>(p, st);
  return pairs <= 2 ? launch_tile<1, 2>(p, st) : pairs <= 4 ? launch_tile<1, 4>(p, st) : pairs <= 8 ? launch_tile<1, 8>(p, st) : launch_tile<1, 16>(p, st);
}

extern "C" int cacheir_b200_talking_device_status(int reset) {
  const int step = device_status_word(g_talking_status, reset != 0), prompt = talking_prompt_status(reset != 0);
  return step != 0 ? step : prompt;
}
