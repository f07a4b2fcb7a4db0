// Latent attention over a paged cache of (latent | rotated key part) rows, sm_100a.
//
// prepare   RMS-norms the latent, turns the rotated parts (rotate-half pairs) and appends one cache row per token.
// simple    any extents, float32 arithmetic: one CTA per (token, head) absorbs the key up-projection into the query,
//           attends over the window in latent space, projects the result up and gates it.
// fast      bf16 tensor cores, flash style, in latent space: all heads share the cached row, so the 16/32/64 rows of a
//           CTA's tile are (token, head) pairs of neighbouring tokens of one sequence. A page of 64 cache rows lands
//           in a two-stage ring, one bulk copy per row (padded shared-memory rows: conflict-free ldmatrix). Eight
//           warps split the scores by 16-row band and key range and the output by band and latent columns. Softmax
//           in float32 with the sink as the initial maximum and denominator. A decode batch too small for the SMs
//           splits the window over CTAs; a second kernel combines the parts.
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
  if (down) {
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
  }
  // one thread per pair (or per unrotated element), so that turning in place is safe
  const int units = half + (a.rot_dim - rot_dims);
  for (int i = threadIdx.x; i < a.heads * units; i += 256) {
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
constexpr int kThreads = 256;

struct FastParams {
  cacheir_b200_latent_args a;
  const __nv_bfloat16* q;      // [rows, heads, kv_rank + rot_dim]
  const float* sink;
  __nv_bfloat16* out;          // [rows, heads, kv_rank]
  float* part_o;               // [splits, rows, heads, kv_rank]
  float* part_ml;              // [splits, rows, heads, 2]
  int heads_per_cta, tokens_per_tile, splits;
  int row_bytes;               // padded shared-memory row
};

constexpr int kProbPitch = 144;          // bytes per row of the probability tile when it has memory of its own
// With 64 rotated dimensions and more, the scores' last use of a key tile frees 128 bytes in each of its 64 rows: the
// probabilities go there and the largest latents fit with 64 query rows.
__host__ __device__ constexpr bool prob_in_keys(int rot_dim) { return rot_dim >= 64; }

template <int MROWS, int RANKMAX>
__global__ void __launch_bounds__(kThreads, 1)
latent_attention_kernel(const FastParams p) {
  constexpr int MW = MROWS / 16;            // 16-row bands
  constexpr int NW = 8 / MW;                // warps per band
  constexpr int NT = 8 / NW;                // 8-key score tiles per warp
  constexpr int PW = (RANKMAX / 16 + NW - 1) / NW;   // 16-column output pairs per warp
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~static_cast<uintptr_t>(127));
  const cacheir_b200_latent_args& a = p.a;
  const int width = a.kv_rank + a.rot_dim;
  const int rb = p.row_bytes;
  uint8_t* s_kv = smem;                                  // [2][64][rb]
  uint8_t* s_q = s_kv + 2 * kPage * rb;                  // [MROWS][rb]
  const bool shared_p = prob_in_keys(a.rot_dim);
  const int pp = shared_p ? rb : kProbPitch;
  uint8_t* s_own_p = s_q + MROWS * rb;                   // [MROWS][kProbPitch], absent when shared_p
  float* s_red = reinterpret_cast<float*>(s_own_p + (shared_p ? 0 : MROWS * kProbPitch));   // [MROWS][NW]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_red + MROWS * NW);          // [2]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int mw = warp / NW, cw = warp % NW;
  const int head0 = blockIdx.y * p.heads_per_cta;
  const int nheads = min(p.heads_per_cta, a.heads - head0);

  int seg, row0, ntok;
  if (a.decode) {
    seg = row0 = static_cast<int>(blockIdx.x);
    ntok = 1;
  } else {
    const RaggedItem it = find_item(a.cu_rows, a.segments, p.tokens_per_tile, blockIdx.x);
    if (it.seg < 0) return;
    seg = it.seg; row0 = it.row0; ntok = it.count;
  }
  const int pos0 = a.positions[row0];
  const int pos_last = pos0 + ntok - 1;
  // pages of this tile's keys, cut evenly over the splits
  const int key_lo = max(0, pos0 - a.window + 1);
  const int page_lo = key_lo / kPage, pages = pos_last / kPage - page_lo + 1;
  const int split = blockIdx.z;
  const int pg_begin = page_lo + pages * split / p.splits, pg_end = page_lo + pages * (split + 1) / p.splits;

  // Q tile: row = token * nheads + head; rows beyond and the k padding are zero
  for (int i = threadIdx.x; i < MROWS * rb / 16; i += kThreads) reinterpret_cast<uint4*>(s_q)[i] = make_uint4(0u, 0u, 0u, 0u);
  for (int i = threadIdx.x; i < 2 * kPage * rb / 16; i += kThreads) reinterpret_cast<uint4*>(s_kv)[i] = make_uint4(0u, 0u, 0u, 0u);
  if (threadIdx.x == 0) {
    ptx::mbar_init(smem_addr(&bars[0]), 1);
    ptx::mbar_init(smem_addr(&bars[1]), 1);
    ptx::mbar_fence_init();
  }
  __syncthreads();
  const int used = ntok * nheads;
  const int chunks = width / 8;
  for (int i = threadIdx.x; i < used * chunks; i += kThreads) {
    const int r = i / chunks, c = i % chunks;
    const size_t src = (static_cast<size_t>(row0 + r / nheads) * a.heads + head0 + r % nheads) * width + c * 8;
    *reinterpret_cast<uint4*>(s_q + r * rb + c * 16) = *reinterpret_cast<const uint4*>(p.q + src);
  }
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");     // zeroed ring rows before the copy engine writes them
  __syncthreads();

  auto load_page = [&](int pg, int stage) {      // warp 0
    const int lo = max(key_lo - pg * kPage, 0), hi = min(pos_last - pg * kPage, kPage - 1);
    const uint32_t bar = smem_addr(&bars[stage]);
    int slot = pg < a.max_pages ? a.page_table[static_cast<size_t>(seg) * a.max_pages + pg] : 0;
    slot = min(max(slot, 0), a.num_slots - 1);
    const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(a.pool) + static_cast<size_t>(slot) * kPage * width;
    if (lane == 0) ptx::mbar_expect_tx(bar, (hi - lo + 1) * width * 2);
    __syncwarp();
    for (int r = lo + lane; r <= hi; r += 32)
      ptx::bulk_load(smem_addr(s_kv + (stage * kPage + r) * rb), src + static_cast<size_t>(r) * width, width * 2, bar);
  };
  if (warp == 0 && pg_begin < pg_end) load_page(pg_begin, 0);

  float acc[PW][2][4];
#pragma unroll
  for (int i = 0; i < PW; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
  // this thread's two rows of the band
  float m_run[2], l_run[2];
  int row_pos[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = mw * 16 + (lane >> 2) + e * 8;
    const bool real = r < used;
    row_pos[e] = real ? pos0 + r / nheads : -1;
    m_run[e] = (real && split == 0) ? p.sink[head0 + r % nheads] * kLog2e : -1e30f;
    l_run[e] = (real && split == 0 && cw == 0 && (lane & 3) == 0) ? 1.f : 0.f;
  }
  const float qscale = a.scale * kLog2e;
  const int ksteps = (width + 15) / 16;
  const int pairs = a.kv_rank / 16;
  const int pair0 = cw * PW;

  bool ok = true;
  for (int pg = pg_begin; pg < pg_end; ++pg) {
    const int it = pg - pg_begin, stage = it & 1;
    if (warp == 0 && pg + 1 < pg_end) load_page(pg + 1, stage ^ 1);
    ok = ptx::mbar_wait(smem_addr(&bars[stage]), (it >> 1) & 1, &g_latent_status, (7 << 8) | 1) && ok;
    const uint32_t kv = smem_addr(s_kv + stage * kPage * rb);
    uint8_t* s_p = shared_p ? s_kv + stage * kPage * rb + a.kv_rank * 2 : s_own_p;
    // scores: 16 rows x (8 NT) keys
    float s[NT][4];
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[t][e] = 0.f;
    const uint32_t qa = smem_addr(s_q) + (mw * 16 + (lane & 15)) * rb + (lane >> 4) * 16;
    const int key0 = cw * NT * 8;
    if constexpr (NT == 1) {
      const uint32_t ka = kv + (key0 + (lane & 7)) * rb + ((lane >> 3) & 1) * 16;
#pragma unroll 4
      for (int k = 0; k < ksteps; ++k) {
        uint32_t af[4], bf[2];
        ldsm_x4(qa + k * 32, af);
        ldsm_x2(ka + k * 32, bf);
        mma_bf16(s[0], af, bf[0], bf[1]);
      }
    } else {
      const uint32_t ka = kv + (key0 + (lane & 7) + ((lane >> 4) << 3)) * rb + ((lane >> 3) & 1) * 16;
#pragma unroll 4
      for (int k = 0; k < ksteps; ++k) {
        uint32_t af[4];
        ldsm_x4(qa + k * 32, af);
#pragma unroll
        for (int t = 0; t < NT; t += 2) {
          uint32_t bf[4];
          ldsm_x4(ka + t * 8 * rb + k * 32, bf);
          mma_bf16(s[t], af, bf[0], bf[1]);
          mma_bf16(s[t + 1], af, bf[2], bf[3]);
        }
      }
    }
    // scale, mask, row maximum
    float mx[2] = {-1e30f, -1e30f};
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = pg * kPage + key0 + t * 8 + (lane & 3) * 2 + (e & 1);
        const int rp = row_pos[e >> 1];
        const bool seen = key <= rp && key > rp - a.window;
        s[t][e] = seen ? s[t][e] * qscale : -INFINITY;
        mx[e >> 1] = fmaxf(mx[e >> 1], s[t][e]);
      }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
      if ((lane & 3) == 0) s_red[(mw * 16 + (lane >> 2) + e * 8) * NW + cw] = mx[e];
    }
    __syncthreads();
    float alpha[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float* red = s_red + (mw * 16 + (lane >> 2) + e * 8) * NW;
      float m_new = m_run[e];
#pragma unroll
      for (int w = 0; w < NW; ++w) m_new = fmaxf(m_new, red[w]);
      alpha[e] = exp2f(m_run[e] - m_new);
      m_run[e] = m_new;
      l_run[e] *= alpha[e];
    }
#pragma unroll
    for (int t = 0; t < NT; ++t) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[t][e] = exp2f(s[t][e] - m_run[e >> 1]);       // masked: exp2(-inf) = 0
        l_run[e >> 1] += s[t][e];
      }
      uint8_t* dst = s_p + (mw * 16 + (lane >> 2)) * pp + (key0 + t * 8 + (lane & 3) * 2) * 2;
      *reinterpret_cast<uint32_t*>(dst) = pack_bf16(s[t][0], s[t][1]);
      *reinterpret_cast<uint32_t*>(dst + 8 * pp) = pack_bf16(s[t][2], s[t][3]);
    }
    __syncthreads();
    // output columns
#pragma unroll
    for (int i = 0; i < PW; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        acc[i][j][0] *= alpha[0]; acc[i][j][1] *= alpha[0];
        acc[i][j][2] *= alpha[1]; acc[i][j][3] *= alpha[1];
      }
    const uint32_t pa = smem_addr(s_p) + (mw * 16 + (lane & 15)) * pp + (lane >> 4) * 16;
    const uint32_t va = kv + ((lane & 7) + ((lane >> 3) & 1) * 8) * rb + (lane >> 4) * 16;
#pragma unroll
    for (int k = 0; k < kPage / 16; ++k) {
      uint32_t af[4];
      ldsm_x4(pa + k * 32, af);
#pragma unroll
      for (int i = 0; i < PW; ++i) {
        if (pair0 + i < pairs) {
          uint32_t bf[4];
          ldsm_x4_t(va + k * 16 * rb + (pair0 + i) * 32, bf);
          mma_bf16(acc[i][0], af, bf[0], bf[1]);
          mma_bf16(acc[i][1], af, bf[2], bf[3]);
        }
      }
    }
    if (shared_p) asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // s_p lies where the next page lands
    __syncthreads();        // the stage, s_p and s_red are free again
  }

  // row sums over the band's warps
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 1);
    l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 2);
    if ((lane & 3) == 0) s_red[(mw * 16 + (lane >> 2) + e * 8) * NW + cw] = l_run[e];
  }
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = mw * 16 + (lane >> 2) + e * 8;
    if (r >= used) continue;
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) l += s_red[r * NW + w];
    const size_t th = static_cast<size_t>(row0 + r / nheads) * a.heads + head0 + r % nheads;
    if (p.splits == 1) {
      const float inv = 1.f / l;
      __nv_bfloat16* dst = p.out + th * a.kv_rank;
#pragma unroll
      for (int i = 0; i < PW; ++i)
        if (pair0 + i < pairs)
#pragma unroll
          for (int j = 0; j < 2; ++j)
            *reinterpret_cast<uint32_t*>(dst + (pair0 + i) * 16 + j * 8 + (lane & 3) * 2) =
                pack_bf16(acc[i][j][e * 2] * inv, acc[i][j][e * 2 + 1] * inv);
    } else {
      const size_t base = static_cast<size_t>(split) * a.rows * a.heads + th;
      float* dst = p.part_o + base * a.kv_rank;
#pragma unroll
      for (int i = 0; i < PW; ++i)
        if (pair0 + i < pairs)
#pragma unroll
          for (int j = 0; j < 2; ++j)
            *reinterpret_cast<float2*>(dst + (pair0 + i) * 16 + j * 8 + (lane & 3) * 2) =
                make_float2(acc[i][j][e * 2], acc[i][j][e * 2 + 1]);
      if (cw == 0 && (lane & 3) == 0) {
        p.part_ml[base * 2] = m_run[e];
        p.part_ml[base * 2 + 1] = l;
      }
    }
  }
}

__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, __nv_bfloat16* __restrict__ out, int splits,
                      size_t units, int rank) {
  const size_t u = blockIdx.x;
  float m = -1e30f;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, part_ml[(s * units + u) * 2]);
  float l = 0.f;
  for (int s = 0; s < splits; ++s) l += part_ml[(s * units + u) * 2 + 1] * exp2f(part_ml[(s * units + u) * 2] - m);
  const float inv = 1.f / l;
  for (int c = threadIdx.x * 4; c < rank; c += 512) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < splits; ++s) {
      const float f = exp2f(part_ml[(s * units + u) * 2] - m);
      const float4 o = *reinterpret_cast<const float4*>(part_o + (s * units + u) * rank + c);
      v.x = fmaf(o.x, f, v.x); v.y = fmaf(o.y, f, v.y); v.z = fmaf(o.z, f, v.z); v.w = fmaf(o.w, f, v.w);
    }
    uint2 raw;
    raw.x = pack_bf16(v.x * inv, v.y * inv);
    raw.y = pack_bf16(v.z * inv, v.w * inv);
    *reinterpret_cast<uint2*>(out + u * rank + c) = raw;
  }
}

int padded_row_bytes(int width) { return (width + 15) / 16 * 32 + 16; }
size_t fast_smem(int mrows, int kv_rank, int rot_dim) {
  const int rb = padded_row_bytes(kv_rank + rot_dim);
  return 128 + static_cast<size_t>(2 * kPage + mrows) * rb + (prob_in_keys(rot_dim) ? 0 : static_cast<size_t>(mrows) * kProbPitch) + static_cast<size_t>(mrows) * 8 * 4 + 64;
}
int head_groups(int heads, bool decode) { const int cap = decode ? 32 : 64; return (heads + cap - 1) / cap; }

template <int MROWS, int RANKMAX>
int launch_fast(const FastParams& p, dim3 grid, cudaStream_t st) {
  const size_t smem = fast_smem(MROWS, p.a.kv_rank, p.a.rot_dim);
  auto kern = latent_attention_kernel<MROWS, RANKMAX>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<grid, kThreads, smem, st>>>(p);
  return launch_status();
}

bool latent_args_ok(const cacheir_b200_latent_args& a) {
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
  if (args->dtype == CACHEIR_B200_F32)
    latent_prepare_kernel<float><<<args->rows, 256, 0, as_stream(stream)>>>(
        *args, static_cast<const float*>(down), down_stride, norm_w, eps, static_cast<const float*>(q), q_stride, static_cast<float*>(q_rot),
        q_rot_stride, q_rot_head_stride, table, rope_positions, rot_dims);
  else if (args->dtype == CACHEIR_B200_BF16)
    latent_prepare_kernel<__nv_bfloat16><<<args->rows, 256, 0, as_stream(stream)>>>(
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
  return dtype == CACHEIR_B200_BF16 && page_size == kPage && kv_rank >= 16 && kv_rank % 16 == 0 && kv_rank <= 512 && rot_dim % 8 == 0 &&
         rot_dim <= 128 && fast_smem(64, kv_rank, rot_dim) <= 227 * 1024 ? 1 : 0;
}

extern "C" int cacheir_b200_latent_attention_splits(int rows, int heads, int window, int max_pages, int page_size) {
  if (rows <= 0 || heads <= 0 || page_size <= 0) return 1;
  const int units = rows * head_groups(heads, true);
  int pages = (window + page_size - 2) / page_size + 1;
  if (pages > max_pages) pages = max_pages;
  int s = kNumSMs / units;
  if (s > pages / 2) s = pages / 2;      // at least two pages each
  return s < 1 ? 1 : (s > 32 ? 32 : s);
}

extern "C" size_t cacheir_b200_latent_attention_workspace_bytes(int rows, int heads, int kv_rank, int splits) {
  if (splits <= 1) return 0;
  return static_cast<size_t>(splits) * rows * heads * (kv_rank + 2) * 4;
}

extern "C" int cacheir_b200_latent_attention(const cacheir_b200_latent_args* args, const void* q, const float* sink, void* out, int splits,
                                             void* workspace, size_t workspace_bytes, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_latent_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!latent_args_ok(a) || !q || !sink || !out || (!a.decode && !a.cu_rows) || (a.decode && a.rows != a.segments)) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_latent_attention_supported(a.kv_rank, a.rot_dim, a.page_size, a.dtype)) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(q, 16) || !aligned_to(a.pool, 16) || !aligned_to(out, 16)) return CACHEIR_B200_EALIGN;
  const bool decode = a.decode != 0;
  if (!decode) splits = 1;
  else if (splits <= 0) splits = cacheir_b200_latent_attention_splits(a.rows, a.heads, a.window, a.max_pages, a.page_size);
  if (splits > 1 && (!workspace || workspace_bytes < cacheir_b200_latent_attention_workspace_bytes(a.rows, a.heads, a.kv_rank, splits)))
    return CACHEIR_B200_EWORKSPACE;
  FastParams p{};
  p.a = a;
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.sink = sink;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.splits = splits;
  p.part_o = static_cast<float*>(workspace);
  p.part_ml = p.part_o ? p.part_o + static_cast<size_t>(splits) * a.rows * a.heads * a.kv_rank : nullptr;
  p.row_bytes = padded_row_bytes(a.kv_rank + a.rot_dim);
  const int groups = head_groups(a.heads, decode);
  p.heads_per_cta = (a.heads + groups - 1) / groups;
  int mrows = 64;
  if (decode) mrows = p.heads_per_cta <= 16 ? 16 : 32;
  p.tokens_per_tile = decode ? 1 : mrows / p.heads_per_cta;
  const int items = decode ? a.rows : ragged_items(a.rows, a.segments, p.tokens_per_tile);
  const dim3 grid(items, groups, splits);
  cudaStream_t st = as_stream(stream);
  int rc;
  if (a.kv_rank <= 128) rc = mrows == 16 ? launch_fast<16, 128>(p, grid, st) : mrows == 32 ? launch_fast<32, 128>(p, grid, st) : launch_fast<64, 128>(p, grid, st);
  else if (a.kv_rank <= 256) rc = mrows == 16 ? launch_fast<16, 256>(p, grid, st) : mrows == 32 ? launch_fast<32, 256>(p, grid, st) : launch_fast<64, 256>(p, grid, st);
  else rc = mrows == 16 ? launch_fast<16, 512>(p, grid, st) : mrows == 32 ? launch_fast<32, 512>(p, grid, st) : launch_fast<64, 512>(p, grid, st);
  if (rc != 0 || splits == 1) return rc;
  latent_combine_kernel<<<a.rows * a.heads, 128, 0, st>>>(p.part_o, p.part_ml, p.out, splits, static_cast<size_t>(a.rows) * a.heads, a.kv_rank);
  return launch_status();
}
