// Latent attention over a paged cache of (latent | rotated key part) rows, sm_100a.
//
// prepare   RMS-norms the latent, turns the rotated parts (rotate-half pairs) and appends one cache row per token.
// simple    any extents, float32 arithmetic: one CTA per (token, head) absorbs the key up-projection into the query,
//           attends over the window in latent space, projects the result up and gates it.
// fast      bf16 tensor cores, flash style, in latent space: all heads share the cached row, so the 16 or 32 rows of a
//           CTA's tile are (token, head) pairs of neighbouring tokens of one sequence. Half pages of 32 cache rows land
//           in a ring as TMA boxes of 64 columns (128-byte swizzle: conflict-free ldmatrix). Softmax in float32
//           with the sink as the initial maximum and denominator. A decode batch too small for the SMs splits the
//           window over the CTAs of a cluster, which combine their parts through distributed shared memory.
#include "hybrid_common.cuh"
#include "ragged.cuh"
#include "tc_ptx.cuh"

namespace cb200 {
namespace {

__device__ int g_latent_status = 0;

constexpr float kLog2e = 1.4426950408889634f;
constexpr int kPage = 64;

template <typename T>
__global__ void __launch_bounds__(256)
latent_prepare_kernel(const cacheir_b200_latent_args a, const T* __restrict__ down, long long down_stride, const float* __restrict__ norm_w,
                      float eps, const T* q, long long q_stride, T* q_rot, long long q_rot_stride, int q_rot_head_stride,
                      const float2* __restrict__ table, int table_positions, int rot_dims) {
  __shared__ float scratch[32];
  const int row = blockIdx.x;
  const int seg = a.row_seg[row];
  if (seg < 0) return;
  const int pos = a.positions[row];
  if (pos < 0 || pos >= table_positions || pos / a.page_size >= a.max_pages) return;
  const float2* cs = table + static_cast<size_t>(pos) * (rot_dims / 2);
  const int half = rot_dims / 2;
  if (down && blockIdx.y == gridDim.y - 1) {      // one CTA of the row writes the cache, the others turn the queries
    const T* d = down + static_cast<size_t>(row) * down_stride;
    const int width = a.kv_rank + a.rot_dim;
    float ss = 0.f;
    for (int c = threadIdx.x; c < a.kv_rank; c += 256) { const float v = Elem<T>::ld(d + c); ss = fmaf(v, v, ss); }
    const float inv = 1.f / sqrtf(block_sum_all(ss, scratch) / static_cast<float>(a.kv_rank) + eps);
    const int slot = a.page_table[static_cast<size_t>(seg) * a.max_pages + pos / a.page_size];
    if (slot >= 0 && slot < a.num_slots) {
      T* dst = static_cast<T*>(a.pool) + (static_cast<size_t>(slot) * a.page_size + pos % a.page_size) * width;
      for (int c = threadIdx.x; c < a.kv_rank; c += 256) Elem<T>::st(dst + c, Elem<T>::ld(d + c) * inv * norm_w[c]);
      for (int c = threadIdx.x; c < a.rot_dim; c += 256) {
        float v = Elem<T>::ld(d + a.kv_rank + c);
        if (c < half) v = v * cs[c].x - Elem<T>::ld(d + a.kv_rank + c + half) * cs[c].y;
        else if (c < rot_dims) v = v * cs[c - half].x + Elem<T>::ld(d + a.kv_rank + c - half) * cs[c - half].y;
        Elem<T>::st(dst + a.kv_rank + c, v);
      }
    }
    return;
  }
  // one thread per pair (or per unrotated element), so that turning in place is safe
  const int units = half + (a.rot_dim - rot_dims);
  const int parts = gridDim.y - (down ? 1 : 0);
  for (int i = blockIdx.y * 256 + threadIdx.x; i < a.heads * units; i += parts * 256) {
    const int h = i / units, u = i % units;
    const T* src = q + static_cast<size_t>(row) * q_stride + static_cast<size_t>(h) * (a.dim + a.rot_dim) + a.dim;
    T* dst = q_rot + static_cast<size_t>(row) * q_rot_stride + static_cast<size_t>(h) * q_rot_head_stride;
    if (u < half) {
      const float x = Elem<T>::ld(src + u), y = Elem<T>::ld(src + u + half);
      const float2 t = cs[u];
      Elem<T>::st(dst + u, x * t.x - y * t.y);
      Elem<T>::st(dst + u + half, y * t.x + x * t.y);
    } else {
      Elem<T>::st(dst + u + half, Elem<T>::ld(src + u + half));
    }
  }
}

// ---- simple form -------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
latent_simple_kernel(const cacheir_b200_latent_args a, const T* __restrict__ q, long long q_stride, const T* __restrict__ uk,
                     const T* __restrict__ uv, const float* __restrict__ sink, const T* __restrict__ gate, long long gate_stride,
                     T* __restrict__ out) {
  extern __shared__ float sm[];
  __shared__ float scratch[32];
  const int width = a.kv_rank + a.rot_dim;
  float* sq = sm;                     // [width] query in latent space | rotated part
  float* so = sq + width;             // [kv_rank]
  float* sp = so + a.kv_rank;         // [128]
  const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int seg = a.row_seg[row];
  if (seg < 0) return;
  const int pos = a.positions[row];
  const T* qh = q + static_cast<size_t>(row) * q_stride + static_cast<size_t>(h) * (a.dim + a.rot_dim);
  for (int r = tid; r < width; r += 128) {
    float v = 0.f;
    if (r < a.kv_rank) {
      for (int d = 0; d < a.dim; ++d) v = fmaf(Elem<T>::ld(qh + d), Elem<T>::ld(uk + (static_cast<size_t>(h) * a.dim + d) * a.kv_rank + r), v);
      so[r] = 0.f;
    } else {
      v = Elem<T>::ld(qh + a.dim + r - a.kv_rank);
    }
    sq[r] = v;
  }
  float m = sink[h], l = 1.f;
  const int lo = max(0, pos - a.window + 1);
  __syncthreads();
  for (int k0 = lo; k0 <= pos; k0 += 128) {
    const int j = k0 + tid;
    float s = -INFINITY;
    if (j <= pos) {
      const int slot = a.page_table[static_cast<size_t>(seg) * a.max_pages + min(j / a.page_size, a.max_pages - 1)];
      const T* kr = static_cast<const T*>(a.pool) + (static_cast<size_t>(min(max(slot, 0), a.num_slots - 1)) * a.page_size + j % a.page_size) * width;
      float dot = 0.f;
      for (int r = 0; r < width; ++r) dot = fmaf(sq[r], Elem<T>::ld(kr + r), dot);
      s = dot * a.scale;
    }
    const float wm = warp_max(s);
    if ((tid & 31) == 0) scratch[tid >> 5] = wm;
    __syncthreads();
    const float m_new = fmaxf(m, fmaxf(fmaxf(scratch[0], scratch[1]), fmaxf(scratch[2], scratch[3])));
    const float p = j <= pos ? expf(s - m_new) : 0.f;
    sp[tid] = p;
    const float alpha = expf(m - m_new);
    l = l * alpha + block_sum_all(p, scratch);      // (its barriers also publish sp)
    m = m_new;
    const int n = min(128, pos - k0 + 1);
    for (int r = tid; r < a.kv_rank; r += 128) {
      float acc = so[r] * alpha;
      for (int i = 0; i < n; ++i) {
        const int jj = k0 + i;
        const int slot = a.page_table[static_cast<size_t>(seg) * a.max_pages + min(jj / a.page_size, a.max_pages - 1)];
        acc = fmaf(sp[i], Elem<T>::ld(static_cast<const T*>(a.pool) +
                                      (static_cast<size_t>(min(max(slot, 0), a.num_slots - 1)) * a.page_size + jj % a.page_size) * width + r), acc);
      }
      so[r] = acc;
    }
    __syncthreads();
  }
  const float inv = 1.f / l;
  for (int v = tid; v < a.vdim; v += 128) {
    float acc = 0.f;
    const T* uvr = uv + (static_cast<size_t>(h) * a.vdim + v) * a.kv_rank;
    for (int r = 0; r < a.kv_rank; ++r) acc = fmaf(so[r], Elem<T>::ld(uvr + r), acc);
    const float g = Elem<T>::ld(gate + static_cast<size_t>(row) * gate_stride + static_cast<size_t>(h) * a.vdim + v);
    Elem<T>::st(out + static_cast<size_t>(row) * a.heads * a.vdim + static_cast<size_t>(h) * a.vdim + v, acc * inv * sigmoid_exact(g));
  }
}

// ---- tensor-core form ----------------------------------------------------------------------------------------------
// 16 warps. Scores: MW bands of 16 rows x KG key groups x 4 quarters of the inner dimension; a warp's part of Q stays in
// registers for the whole kernel. The quarters meet in shared memory, where warp w finishes rows w MW .. w MW + MW - 1
// (scale, mask, running maximum and sum, probabilities as bf16). Output: MW bands x 16/MW groups of latent columns.
constexpr int kThreads = 512;
constexpr int kHalf = kPage / 2;         // the ring moves half pages, so that it prefetches while a page is in use
constexpr int kScorePitch = 72;          // floats: conflict-free for the accumulator layout
constexpr int kProbPitch = 144;          // bytes
constexpr int kMaxSplits = 8;            // CTAs of a cluster
constexpr int kMaxStages = 8;
constexpr int kBoxBytes = kHalf * 128;   // 32 rows x 64 columns

struct FastParams {
  cacheir_b200_latent_args a;
  const __nv_bfloat16* q;      // [rows, heads, kv_rank + rot_dim]
  const float* sink;
  __nv_bfloat16* out;          // [rows, heads, kv_rank]
  int heads_per_cta, tokens_per_tile, splits;
  int boxes;                   // 64-column boxes of a cache row
  int stages;                  // half pages in the ring
  int ring_bytes;              // ring, at least the combine's float tile
};

__device__ __forceinline__ float ld_peer_f32(uint32_t local_addr, uint32_t rank) {
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

// RANKMAX: latent columns the accumulators have room for; KSQ: 16-wide inner steps of a quarter
template <int MW, int RANKMAX, int KSQ>
__global__ void __launch_bounds__(kThreads, 1)
latent_attention_kernel(const __grid_constant__ CUtensorMap tmap, const FastParams p) {
  constexpr int MROWS = MW * 16;
  constexpr int KG = 4 / MW;               // key groups of a page
  constexpr int NT = 8 / KG;               // 8-key score tiles per warp
  constexpr int CW = 16 / MW;              // column groups
  constexpr int PW = (RANKMAX / 16 + CW - 1) / CW;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const cacheir_b200_latent_args& a = p.a;
  const int width = a.kv_rank + a.rot_dim;
  uint8_t* s_kv = smem;                                                      // [stages][boxes][32 rows][128 bytes], swizzled
  const int half_bytes = p.boxes * kBoxBytes;
  float* s_score = reinterpret_cast<float*>(smem + p.ring_bytes);            // [4][MROWS][kScorePitch]
  uint8_t* s_p = reinterpret_cast<uint8_t*>(s_score + 4 * MROWS * kScorePitch);   // [MROWS][kProbPitch]
  float* s_alpha = reinterpret_cast<float*>(s_p + MROWS * kProbPitch);       // [MROWS]
  float* s_ml = s_alpha + MROWS;                                             // [MROWS][2]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_ml + 2 * MROWS);            // [stages]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head0 = blockIdx.y * p.heads_per_cta;
  const int nheads = min(p.heads_per_cta, a.heads - head0);
  const int split = blockIdx.z;            // (the cluster spans the whole z extent)

  int seg, row0, ntok;
  if (a.decode) {
    seg = row0 = static_cast<int>(blockIdx.x);
    ntok = 1;
  } else {
    const RaggedItem it = find_item(a.cu_rows, a.segments, p.tokens_per_tile, blockIdx.x);
    if (it.seg < 0) return;                // (never in a cluster: only decode steps split)
    seg = it.seg; row0 = it.row0; ntok = it.count;
  }
  const int pos0 = a.positions[row0];
  const int pos_last = pos0 + ntok - 1;
  const int used = ntok * nheads;          // tile row = token * nheads + head
  // pages of this tile's keys, cut evenly over the splits
  const int key_lo = max(0, pos0 - a.window + 1);
  const int page_lo = key_lo / kPage, pages = pos_last / kPage - page_lo + 1;
  const int pg_begin = page_lo + pages * split / p.splits;
  const int npages = page_lo + pages * (split + 1) / p.splits - pg_begin;

  auto page_slot = [&](int pg) {
    const int slot = pg < a.max_pages ? a.page_table[static_cast<size_t>(seg) * a.max_pages + pg] : 0;
    return min(max(slot, 0), a.num_slots - 1);
  };
  // One box of a half page. Rows that nobody attends to come along (their probabilities are zero), columns beyond the
  // cache row read as zero.
  auto load_box = [&](int stage, int slot, int half, int box) {
    const uint32_t bar = smem_addr(&bars[stage]);
    if (box == 0) ptx::mbar_expect_tx(bar, half_bytes);
    ptx::tma_load_2d(smem_addr(s_kv + stage * half_bytes + box * kBoxBytes), &tmap, bar, box * 64, slot * kPage + half * kHalf);
  };
  if (threadIdx.x == 0) {
    for (int s = 0; s < p.stages; ++s) ptx::mbar_init(smem_addr(&bars[s]), 1);
    ptx::mbar_fence_init();
  }
  __syncthreads();
  // boxes are dealt over the warps: this warp's lane 0 requests boxes warp, warp + 16 of the 2 * boxes of a page pair
  const int pre = min(p.stages, 2 * npages);
  if (lane == 0)
    for (int b = warp; b < pre * p.boxes; b += 16) {
      const int j = b / p.boxes;
      load_box(j, page_slot(pg_begin + (j >> 1)), j & 1, b - j * p.boxes);
    }
  const int hi_box = warp >= p.boxes ? 1 : 0;      // which of the two halves box `warp` belongs to, box warp + 16 the second
  // half page j = 2 it - 2 + stages (+1) goes where half page 2 it - 2 (+1) was
  int next_slot[2];
#pragma unroll
  for (int u = 0; u < 2; ++u) next_slot[u] = page_slot(pg_begin + ((p.stages + (u ? 1 : hi_box)) >> 1));

  // roles in the score phase
  const int kq = warp & 3, band = (warp >> 2) % MW, kg = (warp >> 2) / MW;
  const int ksteps = (width + 15) / 16;
  const int k_begin = ksteps * kq / 4, k_count = ksteps * (kq + 1) / 4 - k_begin;
  uint32_t qf[KSQ][4];
#pragma unroll
  for (int k = 0; k < KSQ; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = band * 16 + (lane >> 2) + (e & 1) * 8, c = (k_begin + k) * 16 + (lane & 3) * 2 + (e >> 1) * 8;
      qf[k][e] = (k < k_count && r < used && c < width)
                     ? *reinterpret_cast<const uint32_t*>(p.q + (static_cast<size_t>(row0 + r / nheads) * a.heads + head0 + r % nheads) * width + c)
                     : 0u;
    }
  // roles in the softmax phase: rows warp * MW + i
  float m_run[MW], l_run[MW];
  int row_pos[MW];
#pragma unroll
  for (int i = 0; i < MW; ++i) {
    const int r = warp * MW + i;
    const bool real = r < used;
    row_pos[i] = real ? pos0 + r / nheads : -1;
    m_run[i] = (real && split == 0) ? p.sink[head0 + r % nheads] * kLog2e : -1e30f;
    l_run[i] = (real && split == 0 && lane == 0) ? 1.f : 0.f;
  }
  const float qscale = a.scale * kLog2e;
  // roles in the output phase
  const int oband = warp % MW, cw = warp / MW;
  const int pairs = a.kv_rank / 16, pair0 = cw * PW;
  float acc[PW][2][4];
#pragma unroll
  for (int i = 0; i < PW; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;

  int free0 = 0, free1 = 0;                // stages of the previous page
  int st0 = 0, parity0 = 0;                // stage and phase of the current page's first half
  for (int it = 0; it < npages; ++it) {
    const bool wrap1 = st0 + 1 == p.stages;
    const int st1 = wrap1 ? 0 : st0 + 1, parity1 = parity0 ^ (wrap1 ? 1 : 0);
    ptx::mbar_wait(smem_addr(&bars[st0]), parity0, &g_latent_status, (7 << 8) | 1);
    ptx::mbar_wait(smem_addr(&bars[st1]), parity1, &g_latent_status, (7 << 8) | 2);
    const uint32_t kv0 = smem_addr(s_kv) + st0 * half_bytes, kv1 = smem_addr(s_kv) + st1 * half_bytes;
    {
      float s[NT][4];
#pragma unroll
      for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[t][e] = 0.f;
      const int key0 = kg * NT * 8;        // a group lies inside one half
      const uint32_t ka = (key0 < kHalf ? kv0 : kv1) + ((key0 % kHalf) + (lane & 7) + ((lane >> 4) << 3)) * 128;
#pragma unroll
      for (int k = 0; k < KSQ; ++k) {
        if (k < k_count) {                  // (the same for all warps up to one step)
          const int chunk = 2 * (k_begin + k) + ((lane >> 3) & 1);        // 16-byte pieces of the row
          const uint32_t kc = ka + (chunk >> 3) * kBoxBytes + (((chunk ^ lane) & 7) << 4);
#pragma unroll
          for (int t = 0; t < NT; t += 2) {
            uint32_t bf[4];
            ldsm_x4(kc + t * 8 * 128, bf);
            mma_bf16(s[t], qf[k], bf[0], bf[1]);
            mma_bf16(s[t + 1], qf[k], bf[2], bf[3]);
          }
        }
      }
      float* dst = s_score + (kq * MROWS + band * 16 + (lane >> 2)) * kScorePitch + key0 + (lane & 3) * 2;
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        *reinterpret_cast<float2*>(dst + t * 8) = make_float2(s[t][0], s[t][1]);
        *reinterpret_cast<float2*>(dst + 8 * kScorePitch + t * 8) = make_float2(s[t][2], s[t][3]);
      }
    }
    __syncthreads();                       // scores complete; everyone has left the previous page
    if (it > 0) {                          // the previous page's halves are free: every warp requests a box or two
      const int j0 = 2 * it - 2 + p.stages;
      if (lane == 0) {
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int b = warp + 16 * u, h = u ? 1 : hi_box;
          if (b < 2 * p.boxes && j0 + h < 2 * npages) load_box(h ? free1 : free0, next_slot[u], (j0 + h) & 1, b - h * p.boxes);
        }
      }
#pragma unroll
      for (int u = 0; u < 2; ++u) next_slot[u] = page_slot(pg_begin + ((j0 + 2 + (u ? 1 : hi_box)) >> 1));
    }
    free0 = st0;
    free1 = st1;
    st0 = st1 + 1 == p.stages ? 0 : st1 + 1;
    parity0 = parity1 ^ (st0 == 0 ? 1 : 0);
    const int key = (pg_begin + it) * kPage + lane * 2;
    float2 v[MW];
    float mx[MW], alpha[MW];
#pragma unroll
    for (int i = 0; i < MW; ++i) v[i] = *reinterpret_cast<const float2*>(s_score + (warp * MW + i) * kScorePitch + lane * 2);
#pragma unroll
    for (int part = 1; part < 4; ++part)
#pragma unroll
      for (int i = 0; i < MW; ++i) {
        const float2 x = *reinterpret_cast<const float2*>(s_score + (part * MROWS + warp * MW + i) * kScorePitch + lane * 2);
        v[i].x += x.x; v[i].y += x.y;
      }
#pragma unroll
    for (int i = 0; i < MW; ++i) {
      v[i].x = (key <= row_pos[i] && key > row_pos[i] - a.window) ? v[i].x * qscale : -INFINITY;
      v[i].y = (key + 1 <= row_pos[i] && key + 1 > row_pos[i] - a.window) ? v[i].y * qscale : -INFINITY;
      mx[i] = fmaxf(v[i].x, v[i].y);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1)
#pragma unroll
      for (int i = 0; i < MW; ++i) mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], off));
#pragma unroll
    for (int i = 0; i < MW; ++i) {
      const int r = warp * MW + i;
      mx[i] = fmaxf(mx[i], m_run[i]);
      alpha[i] = exp2f(m_run[i] - mx[i]);
      v[i].x = exp2f(v[i].x - mx[i]);
      v[i].y = exp2f(v[i].y - mx[i]);
      m_run[i] = mx[i];
      *reinterpret_cast<uint32_t*>(s_p + r * kProbPitch + lane * 4) = pack_bf16(v[i].x, v[i].y);
      if (lane == 0) s_alpha[r] = alpha[i];
      l_run[i] = fmaf(l_run[i], alpha[i], v[i].x + v[i].y);
    }
    __syncthreads();                       // probabilities complete
    const float f0 = s_alpha[oband * 16 + (lane >> 2)], f1 = s_alpha[oband * 16 + (lane >> 2) + 8];
    if (__any_sync(0xffffffffu, f0 != 1.f || f1 != 1.f)) {
#pragma unroll
      for (int i = 0; i < PW; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          acc[i][j][0] *= f0; acc[i][j][1] *= f0;
          acc[i][j][2] *= f1; acc[i][j][3] *= f1;
        }
    }
    const uint32_t pa = smem_addr(s_p) + (oband * 16 + (lane & 15)) * kProbPitch + (lane >> 4) * 16;
    const uint32_t voff = ((lane & 7) + ((lane >> 3) & 1) * 8) * 128;
#pragma unroll
    for (int k = 0; k < kPage / 16; ++k) {
      uint32_t af[4], bf[PW][4];
      ldsm_x4(pa + k * 32, af);
      const uint32_t va = (k < 2 ? kv0 : kv1) + (k & 1) * 16 * 128 + voff;
#pragma unroll
      for (int i = 0; i < PW; ++i) {
        const int chunk = 2 * min(pair0 + i, pairs - 1) + (lane >> 4);      // (columns beyond the latent are not stored)
        ldsm_x4_t(va + (chunk >> 3) * kBoxBytes + (((chunk ^ lane) & 7) << 4), bf[i]);
      }
#pragma unroll
      for (int i = 0; i < PW; ++i) {
        mma_bf16(acc[i][0], af, bf[i][0], bf[i][1]);
        mma_bf16(acc[i][1], af, bf[i][2], bf[i][3]);
      }
    }
  }

  // row sums and maxima
#pragma unroll
  for (int i = 0; i < MW; ++i) {
    const float l = warp_sum(l_run[i]);
    if (lane == 0) {
      s_ml[(warp * MW + i) * 2] = m_run[i];
      s_ml[(warp * MW + i) * 2 + 1] = l;
    }
  }
  __syncthreads();                         // (also: the ring is free)
  if (p.splits == 1) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = oband * 16 + (lane >> 2) + e * 8;
      if (r >= used) continue;
      const float inv = 1.f / s_ml[r * 2 + 1];
      __nv_bfloat16* dst = p.out + (static_cast<size_t>(row0 + r / nheads) * a.heads + head0 + r % nheads) * a.kv_rank + (lane & 3) * 2;
#pragma unroll
      for (int i = 0; i < PW; ++i)
        if (pair0 + i < pairs)
#pragma unroll
          for (int j = 0; j < 2; ++j)
            *reinterpret_cast<uint32_t*>(dst + (pair0 + i) * 16 + j * 8) = pack_bf16(acc[i][j][e * 2] * inv, acc[i][j][e * 2 + 1] * inv);
    }
    return;
  }
  // the cluster's CTAs share one tile: partial outputs in shared memory, rows dealt out, parts added in rank order
  const int opitch = a.kv_rank + 8;
  float* s_o = reinterpret_cast<float*>(smem);
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    float* dst = s_o + (oband * 16 + (lane >> 2) + e * 8) * opitch + (lane & 3) * 2;
#pragma unroll
    for (int i = 0; i < PW; ++i)
      if (pair0 + i < pairs)
#pragma unroll
        for (int j = 0; j < 2; ++j)
          *reinterpret_cast<float2*>(dst + (pair0 + i) * 16 + j * 8) = make_float2(acc[i][j][e * 2], acc[i][j][e * 2 + 1]);
  }
  cluster_sync_all();
  for (int r = split; r < used; r += p.splits) {
    float m[kMaxSplits], top = -1e30f, l = 0.f;
#pragma unroll
    for (int s = 0; s < kMaxSplits; ++s) {
      m[s] = s < p.splits ? ld_peer_f32(smem_addr(s_ml + r * 2), s) : -1e30f;
      top = fmaxf(top, m[s]);
    }
#pragma unroll
    for (int s = 0; s < kMaxSplits; ++s) {
      m[s] = exp2f(m[s] - top);
      if (s < p.splits) l = fmaf(ld_peer_f32(smem_addr(s_ml + r * 2 + 1), s), m[s], l);
    }
    const float inv = 1.f / l;
    __nv_bfloat16* dst = p.out + (static_cast<size_t>(row0 + r / nheads) * a.heads + head0 + r % nheads) * a.kv_rank;
    for (int c = threadIdx.x; c < a.kv_rank; c += kThreads) {
      float v = 0.f;
#pragma unroll
      for (int s = 0; s < kMaxSplits; ++s)
        if (s < p.splits) v = fmaf(ld_peer_f32(smem_addr(s_o + r * opitch + c), s), m[s], v);
      dst[c] = __float2bfloat16_rn(v * inv);
    }
  }
  cluster_sync_all();                      // nobody leaves while its part is being read
}

int row_boxes(int width) { return (width + 63) / 64; }
// shared memory beside the ring
size_t fast_fixed_smem(int mrows) { return 1024 + static_cast<size_t>(mrows) * (4 * kScorePitch * 4 + kProbPitch + 12) + 16 + kMaxStages * 8; }
constexpr size_t kSmemLimit = 227 * 1024;
int fast_stages(int mrows, int width) {
  const int s = static_cast<int>((kSmemLimit - fast_fixed_smem(mrows)) / (static_cast<size_t>(row_boxes(width)) * kBoxBytes));
  return s > kMaxStages ? kMaxStages : s;
}
int head_groups(int heads) { return (heads + 31) / 32; }

bool encode_pool(CUtensorMap* map, const void* base, uint64_t width, uint64_t rows) {
  ptx::EncodeTiledFn fn = ptx::tensor_map_encoder();
  if (!fn) return false;
  const cuuint64_t dims[2] = {width, rows};
  const cuuint64_t strides[1] = {width * 2};
  const cuuint32_t box[2] = {64, kHalf};
  const cuuint32_t elem_strides[2] = {1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem_strides,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int MW, int RANKMAX, int KSQ>
int launch_fast(FastParams p, dim3 grid, cudaStream_t st) {
  const int width = p.a.kv_rank + p.a.rot_dim;
  p.stages = fast_stages(MW * 16, width);
  const size_t ring = static_cast<size_t>(p.stages) * p.boxes * kBoxBytes, combine = static_cast<size_t>(MW) * 16 * (p.a.kv_rank + 8) * 4;
  p.ring_bytes = static_cast<int>(((p.splits > 1 && combine > ring ? combine : ring) + 15) / 16 * 16);
  const size_t smem = p.ring_bytes + fast_fixed_smem(MW * 16);
  if (p.stages < 4 || smem > kSmemLimit) return CACHEIR_B200_EUNSUPPORTED;
  CUtensorMap tmap;
  if (!encode_pool(&tmap, p.a.pool, width, static_cast<uint64_t>(p.a.num_slots) * kPage)) return CACHEIR_B200_EUNSUPPORTED;
  auto kern = latent_attention_kernel<MW, RANKMAX, KSQ>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(kThreads, 1, 1);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = p.splits;
  cfg.attrs = attr;
  cfg.numAttrs = p.splits > 1 ? 1 : 0;
  e = cudaLaunchKernelEx(&cfg, kern, tmap, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  return launch_status();
}

template <int MW>
int launch_fast_size(const FastParams& p, dim3 grid, cudaStream_t st) {
  const int width = p.a.kv_rank + p.a.rot_dim;
  if (p.a.kv_rank <= 128 && width <= 192) return launch_fast<MW, 128, 3>(p, grid, st);
  if (p.a.kv_rank <= 256 && width <= 320) return launch_fast<MW, 256, 5>(p, grid, st);
  if (width <= 576) return launch_fast<MW, 512, 9>(p, grid, st);
  return launch_fast<MW, 512, 10>(p, grid, st);
}

bool latent_args_ok(
const cacheir_b200_latent_args& a) {
  return a.positions && a.row_seg && a.page_table && a.pool && a.segments > 0 && a.max_pages > 0 && a.page_size > 0 && a.num_slots > 0 &&
         a.heads > 0 && a.dim > 0 && a.rot_dim >= 0 && a.vdim > 0 && a.kv_rank > 0 && a.window > 0 && a.heads <= 65535;
}

}  // namespace

int latent_attention_device_status(bool reset) {
  int status = 0;
  if (cudaMemcpyFromSymbol(&status, g_latent_status, sizeof(int)) != cudaSuccess) return -1;
  if (reset && status != 0) {
    const int zero = 0;
    cudaMemcpyToSymbol(g_latent_status, &zero, sizeof(int));
  }
  return status;
}

}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_latent_prepare(const cacheir_b200_latent_args* args, const void* down, long long down_stride,
                                           const float* norm_w, float eps, const void* q, long long q_stride, void* q_rot,
                                           long long q_rot_stride, int q_rot_head_stride, const float* rope_table, int rope_positions,
                                           int rot_dims, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  if (args->rows <= 0) return 0;
  if (!latent_args_ok(*args) || !q || !q_rot || !rope_table || rope_positions <= 0 || rot_dims < 0 || rot_dims % 2 != 0 ||
      rot_dims > args->rot_dim || (down && !norm_w))
    return CACHEIR_B200_EINVAL;
  const float2* table = reinterpret_cast<const float2*>(rope_table);
  const int pairs = args->heads * (args->rot_dim - rot_dims / 2);
  const int parts = args->rows >= kNumSMs ? 1 : (pairs + 255) / 256 < 4 ? (pairs + 255) / 256 : 4;
  const dim3 grid(args->rows, parts + (down ? 1 : 0));
  if (args->dtype == CACHEIR_B200_F32)
    latent_prepare_kernel<float><<<grid, 256, 0, as_stream(stream)>>>(
        *args, static_cast<const float*>(down), down_stride, norm_w, eps, static_cast<const float*>(q), q_stride, static_cast<float*>(q_rot),
        q_rot_stride, q_rot_head_stride, table, rope_positions, rot_dims);
  else if (args->dtype == CACHEIR_B200_BF16)
    latent_prepare_kernel<__nv_bfloat16><<<grid, 256, 0, as_stream(stream)>>>(
        *args, static_cast<const __nv_bfloat16*>(down), down_stride, norm_w, eps, static_cast<const __nv_bfloat16*>(q), q_stride,
        static_cast<__nv_bfloat16*>(q_rot), q_rot_stride, q_rot_head_stride, table, rope_positions, rot_dims);
  else
    return CACHEIR_B200_EUNSUPPORTED;
  return launch_status();
}

extern "C" int cacheir_b200_latent_attention_simple(const cacheir_b200_latent_args* args, const void* q, long long q_stride,
                                                    const void* uk, const void* uv, const float* sink, const void* gate,
                                                    long long gate_stride, void* out, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  if (args->rows <= 0) return 0;
  if (!latent_args_ok(*args) || !q || !uk || !uv || !sink || !gate || !out) return CACHEIR_B200_EINVAL;
  const size_t smem = static_cast<size_t>(2 * args->kv_rank + args->rot_dim + 128) * 4;
  if (smem > 48 * 1024) return CACHEIR_B200_ELIMIT;
  const dim3 grid(args->rows, args->heads);
#define CB200_LATENT_SIMPLE(T)                                                                                              \
  latent_simple_kernel<T><<<grid, 128, smem, as_stream(stream)>>>(*args, static_cast<const T*>(q), q_stride, static_cast<const T*>(uk), \
      static_cast<const T*>(uv), sink, static_cast<const T*>(gate), gate_stride, static_cast<T*>(out))
  if (args->dtype == CACHEIR_B200_F32) CB200_LATENT_SIMPLE(float);
  else if (args->dtype == CACHEIR_B200_BF16) CB200_LATENT_SIMPLE(__nv_bfloat16);
  else return CACHEIR_B200_EUNSUPPORTED;
#undef CB200_LATENT_SIMPLE
  return launch_status();
}

extern "C" int cacheir_b200_latent_attention_supported(int kv_rank, int rot_dim, int page_size, int dtype) {
  return dtype == CACHEIR_B200_BF16 && page_size == kPage && kv_rank >= 16 && kv_rank % 16 == 0 && kv_rank <= 512 && rot_dim >= 0 &&
         rot_dim % 8 == 0 && kv_rank + rot_dim <= 640 && fast_stages(32, kv_rank + rot_dim) >= 4 ? 1 : 0;
}

extern "C" int cacheir_b200_latent_attention_splits(int rows, int heads, int window, int max_pages, int page_size) {
  if (rows <= 0 || heads <= 0 || page_size <= 0) return 1;
  const int units = rows * head_groups(heads);
  int pages = (window + page_size - 2) / page_size + 1;
  if (pages > max_pages) pages = max_pages;
  int s = kNumSMs / units;
  if (s > pages / 2) s = pages / 2;      // at least two pages each
  return s < 1 ? 1 : (s > kMaxSplits ? kMaxSplits : s);
}

extern "C" int cacheir_b200_latent_attention(const cacheir_b200_latent_args* args, const void* q, const float* sink, void* out, int splits,
                                             void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_latent_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!latent_args_ok(a) || !q || !sink || !out || (!a.decode && !a.cu_rows) || (a.decode && a.rows != a.segments)) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_latent_attention_supported(a.kv_rank, a.rot_dim, a.page_size, a.dtype)) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(q, 16) || !aligned_to(a.pool, 16) || !aligned_to(out, 16)) return CACHEIR_B200_EALIGN;
  const bool decode = a.decode != 0;
  if (!decode) splits = 1;
  else if (splits <= 0) splits = cacheir_b200_latent_attention_splits(a.rows, a.heads, a.window, a.max_pages, a.page_size);
  if (splits > kMaxSplits) return CACHEIR_B200_ELIMIT;
  FastParams p{};
  p.a = a;
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.sink = sink;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.splits = splits;
  p.boxes = row_boxes(a.kv_rank + a.rot_dim);
  const int groups = head_groups(a.heads);
  p.heads_per_cta = (a.heads + groups - 1) / groups;
  const bool narrow = decode && p.heads_per_cta <= 16;
  p.tokens_per_tile = decode ? 1 : 32 / p.heads_per_cta;
  const int items = decode ? a.rows : ragged_items(a.rows, a.segments, p.tokens_per_tile);
  const dim3 grid(items, groups, splits);
  return narrow ? launch_fast_size<1>(p, grid, as_stream(stream)) : launch_fast_size<2>(p, grid, as_stream(stream));
}
