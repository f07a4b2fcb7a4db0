// Latent attention over a paged cache of (latent | rotated key part) rows, sm_100a.
//
// prepare   RMS-norms the latent, turns the rotated parts (rotate-half pairs) and appends one cache row per token.
// simple    any extents, float32 arithmetic: one CTA per (token, head) absorbs the key up-projection into the query,
//           attends over the window in latent space, projects the result up and gates it.
// fast      bf16, 5th-generation tensor cores, in latent space: all heads share the cached row, so the 32 or 64 rows of a
//           CTA's tile are (token, head) pairs of neighbouring tokens of one sequence. Pages of 64 cache rows land in a
//           ring as TMA boxes of 64 columns and serve as keys and, read the other way, as values. Softmax in float32
//           with the sink as the initial maximum and denominator. A decode batch too small for the SMs splits the
//           window over the CTAs of a cluster, which combine their parts through distributed shared memory.
#include "cacheir_b200_hybrid.h"
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
// Per 64-key page:   S [rows, keys] = Q K^T          A = the query tile (M 64), B = the page (N 64)
//                    O^T [latent, rows] += V^T P^T   A = the same page read MN-major (M 128 latent columns), B = P
// so the page is used twice as it lies in shared memory and the probabilities go back as the K-major operand that a row's
// threads write. O^T stays in tensor memory. Its columns are rescaled only when a row's maximum has grown by more than
// 2^8 since its reference was chosen (a stale reference costs nothing: numerator and denominator share it).
//   warps 0..7  softmax (lane quarter = warp % 4, key half = warp / 4), rescaling, output
//   warp 8      MMA issue, tensor memory           warp 9  copies
constexpr int kThreads = 320;
constexpr int kSoftThreads = 256;
constexpr int kMaxSplits = 8;            // CTAs of a cluster
constexpr int kMaxStages = 6;            // pages in the ring
constexpr int kBoxBytes = kPage * 128;   // 64 rows x 64 columns
constexpr float kStale = 8.f;

struct FastParams {
  cacheir_b200_latent_args a;
  const float* sink;
  __nv_bfloat16* out;          // [rows, heads, kv_rank]
  int heads_per_cta, tokens_per_tile, splits;
  int boxes;                   // 64-column boxes of a cache row
  int blocks;                  // 128-column blocks of the latent
  int stages;
  int ahead;                   // three pages in the ring: the next page's scores are issued before this page's output
  int p_in_page;               // probabilities overwrite the page's box of rotated key parts, which the scores are done with
  int tmem_cols;
};

__device__ __forceinline__ float ld_peer_f32(uint32_t local_addr, uint32_t rank) {
  uint32_t remote;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local_addr), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote));
  return v;
}
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// Executed by a whole warp so that the operands stay in uniform registers; `lead` picks the issuing lane. Descriptors come as
// their two words: only the address word changes.
__device__ __forceinline__ void mma_f16_ss(uint32_t lead, uint32_t tmem_d, uint32_t a_lo, uint32_t a_hi, uint32_t b_lo, uint32_t b_hi,
                                           uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t.reg .b64 a, b;\n\t"
      "mov.b64 a, {%1, %2};\n\t"
      "mov.b64 b, {%3, %4};\n\t"
      "setp.ne.b32 p, %6, 0;\n\t"
      "setp.ne.b32 q, %7, 0;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], a, b, %5, p;\n\t}"
      ::"r"(tmem_d), "r"(a_lo), "r"(a_hi), "r"(b_lo), "r"(b_hi), "r"(idesc), "r"(accumulate), "r"(lead) : "memory");
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// MN-major operand as 128-byte swizzled rows: 64 columns a box, `box` bytes between boxes, 8-row groups 1024 bytes apart
__device__ __forceinline__ uint64_t smem_desc_mn_sw128(uint32_t addr, uint32_t box) {
  return static_cast<uint64_t>((addr >> 4) & 0x3FFF) | static_cast<uint64_t>((box >> 4) & 0x3FFF) << 16 |
         static_cast<uint64_t>(1024 >> 4) << 32 | static_cast<uint64_t>(1) << 46 | static_cast<uint64_t>(2) << 61;
}
// 16 lanes x 32 columns in the warp-MMA accumulator order: v[4 j + e] = row lane / 4 + 8 (e / 2), column 8 j + 2 (lane % 4) + e % 2
__device__ __forceinline__ void tmem_ld_rows16(uint32_t taddr, float (&v)[16]) {
  uint32_t r[16];
  asm volatile(
      "tcgen05.ld.sync.aligned.16x256b.x4.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
        "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr) : "memory");
  ptx::tc_wait_ld();
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
}
__device__ __forceinline__ void tmem_ld_x16(uint32_t taddr, float (&v)[16]) {
  uint32_t r[16];
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
        "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr) : "memory");
  ptx::tc_wait_ld();
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
}
__device__ __forceinline__ void tmem_st_x16(uint32_t taddr, const float (&v)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "f"(v[0]), "f"(v[1]), "f"(v[2]), "f"(v[3]), "f"(v[4]), "f"(v[5]), "f"(v[6]), "f"(v[7]), "f"(v[8]), "f"(v[9]), "f"(v[10]),
      "f"(v[11]), "f"(v[12]), "f"(v[13]), "f"(v[14]), "f"(v[15]) : "memory");
}
// true in all softmax threads if `p` holds in one of them
__device__ __forceinline__ bool any_softmax(bool p) {
  uint32_t out;
  asm volatile(
      "{\n\t.reg .pred a, b;\n\t"
      "setp.ne.u32 a, %1, 0;\n\t"
      "barrier.cta.red.or.pred b, 1, %2, a;\n\t"
      "selp.u32 %0, 1, 0, b;\n\t}"
      : "=r"(out) : "r"(static_cast<uint32_t>(p)), "n"(kSoftThreads) : "memory");
  return out != 0;
}
__device__ __forceinline__ void sync_softmax() { asm volatile("barrier.cta.sync 1, %0;" ::"n"(kSoftThreads) : "memory"); }

template <int NR>
__global__ void __launch_bounds__(kThreads, 1)
latent_attention_kernel(const __grid_constant__ CUtensorMap tmap_kv, const __grid_constant__ CUtensorMap tmap_q, const FastParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const cacheir_b200_latent_args& a = p.a;
  const int page_bytes = p.boxes * kBoxBytes;
  uint8_t* s_kv = smem;                                         // [stages][boxes][64 rows][128 bytes], swizzled
  uint8_t* s_q = s_kv + p.stages * page_bytes;                  // [boxes][NR rows][128 bytes], swizzled
  uint8_t* s_p = s_q + p.boxes * NR * 128;                      // [2][NR rows][128 bytes], swizzled; absent with p_in_page
  float* s_alpha = reinterpret_cast<float*>(s_p + (p.p_in_page ? 0 : 2 * NR * 128));   // [NR]
  float* s_max = s_alpha + NR;                                  // [2 pages][2 key halves][NR]
  float* s_ml = s_max + 4 * NR;                                 // [NR] references, [NR] denominators
  float* s_w = reinterpret_cast<float*>(s_q);                   // [rows][kMaxSplits][2]: what the combine weighs with (over the queries)
  uint64_t* full = reinterpret_cast<uint64_t*>(s_ml + 2 * NR);  // [stages] a page has landed
  uint64_t* empty = full + kMaxStages;                          // [stages] its output MMAs have retired
  uint64_t* bar_q = empty + kMaxStages;
  uint64_t* bar_s = bar_q + 1;                                  // [2] scores in tensor memory
  uint64_t* bar_p = bar_s + 2;                                  // [2] probabilities in shared memory
  uint64_t* bar_o = bar_p + 2;                                  // the output MMAs of one more page have retired
  uint64_t* bar_done = bar_o + 1;                               // all output MMAs have retired
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar_done + 1);

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
  const int used = ntok * nheads;          // tile row = token * nheads + head: neighbouring rows of q
  // pages of this tile's keys, cut evenly over the splits
  const int key_lo = max(0, pos0 - a.window + 1);
  const int page_lo = key_lo / kPage, pages = pos_last / kPage - page_lo + 1;
  const int pg_begin = page_lo + pages * split / p.splits;
  const int npages = page_lo + pages * (split + 1) / p.splits - pg_begin;

  // The copy warp sets the barriers up and requests the first pages before the block meets.
  int stage = 0, phase = 1;                // its place in the ring
  auto page_row = [&](int it) {            // the page's first row in the pool
    const int pg = pg_begin + it;
    const int slot = pg < a.max_pages ? a.page_table[static_cast<size_t>(seg) * a.max_pages + pg] : 0;
    return min(max(slot, 0), a.num_slots - 1) * kPage;
  };
  auto prefetch_page = [&](int it) {       // into L2, before the ring has room
    if (it >= npages || !a.decode) return;       // (a prompt's tiles find their pages there)
    const int row = page_row(it);
    for (int b = 0; b < p.boxes; ++b)
      asm volatile("cp.async.bulk.prefetch.tensor.2d.L2.global [%0, {%1, %2}];"
                   ::"l"(reinterpret_cast<uint64_t>(&tmap_kv)), "r"(b * 64), "r"(row) : "memory");
  };
  auto load_page = [&](int it) {
    const int row = page_row(it);
    const uint32_t bar = smem_addr(&full[stage]);
    ptx::mbar_expect_tx(bar, page_bytes);
    for (int b = 0; b < p.boxes; ++b)
      ptx::tma_load_2d(smem_addr(s_kv + stage * page_bytes + b * kBoxBytes), &tmap_kv, bar, b * 64, row);
    if (++stage == p.stages) { stage = 0; phase ^= 1; }
  };
  const int first = min(npages, p.stages);
  if (warp == 9 && lane == 0) {
    for (int s = 0; s < p.stages; ++s) { ptx::mbar_init(smem_addr(&full[s]), 1); ptx::mbar_init(smem_addr(&empty[s]), 1); }
    ptx::mbar_init(smem_addr(bar_q), 1);
    for (int s = 0; s < 2; ++s) { ptx::mbar_init(smem_addr(&bar_s[s]), 1); ptx::mbar_init(smem_addr(&bar_p[s]), kSoftThreads); }
    ptx::mbar_init(smem_addr(bar_o), 1);
    ptx::mbar_init(smem_addr(bar_done), 1);
    ptx::mbar_fence_init();
    if (npages > 0) {
      ptx::mbar_expect_tx(smem_addr(bar_q), p.boxes * NR * 128);
      for (int b = 0; b < p.boxes; ++b)
        ptx::tma_load_2d(smem_addr(s_q + b * NR * 128), &tmap_q, smem_addr(bar_q), b * 64, row0 * a.heads + head0);
      for (int it = 0; it < first; ++it) load_page(it);
      for (int it = first; it < first + 2; ++it) prefetch_page(it);
    }
  }
  __syncwarp();
  if (warp == 8) ptx::tc_alloc(smem_addr(tmem_slot), p.tmem_cols);
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t tmem_s = tmem + p.blocks * NR;       // scores: two buffers of 64 columns behind the output blocks
  bool ok = true;

  if (warp == 9) {
    // ---------------- copies ----------------
    if (lane == 0 && npages > 0) {
      for (int it = first; it < npages; ++it) {
        ok = ok && ptx::mbar_wait(smem_addr(&empty[stage]), phase, &g_latent_status, (7 << 8) | 1);
        if (!ok) break;
        load_page(it);
        prefetch_page(it + 2);
      }
      // nothing may still be on its way when the block ends, also after a wait that gave up
      ptx::mbar_wait(smem_addr(bar_q), 0, &g_latent_status, (7 << 8) | 8);
      if (!ok)
        for (int s = 0; s < p.stages; ++s) ptx::mbar_wait(smem_addr(&full[s]), s < stage ? phase ^ 1 : phase, &g_latent_status, (7 << 8) | 9);
    }
    __syncwarp();
  } else if (warp == 8) {
    // ---------------- MMA issue ----------------
    if (npages > 0) {
      const uint32_t lead = lane == 0 ? 1u : 0u;
      const uint32_t id_s = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kPage >> 3) << 17) | (static_cast<uint32_t>(64 >> 4) << 24);
      const uint32_t id_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 15) | (static_cast<uint32_t>(NR >> 3) << 17) |
                            (static_cast<uint32_t>(128 >> 4) << 24);
      const uint64_t dq = ptx::smem_desc_sw128(smem_addr(s_q)), dk = ptx::smem_desc_sw128(smem_addr(s_kv));
      const uint64_t dp = ptx::smem_desc_sw128(smem_addr(p.p_in_page ? s_kv + 2 * p.blocks * kBoxBytes : s_p));
      const uint64_t dv = smem_desc_mn_sw128(smem_addr(s_kv), kBoxBytes);
      const uint32_t k_hi = static_cast<uint32_t>(dk >> 32), v_hi = static_cast<uint32_t>(dv >> 32);     // (dq, dk, dp share theirs)
      const uint32_t stage_step = static_cast<uint32_t>(page_bytes >> 4);
      int s_stage = 0, s_phase = 0, o_stage = 0;
      int next_s = 0, next_o = 0;            // next page to score, next page to add to the output
      bool fill = true;
      ok = ptx::mbar_wait(smem_addr(bar_q), 0, &g_latent_status, (7 << 8) | 3);
      // Two pages are scored before the first one's output, so that softmax runs beside MMAs. With a ring of two pages they go
      // pair by pair: the second page's output overlaps the next pair's loads.
#pragma unroll 1
      while (next_o < npages) {
        if (next_s < npages && (p.ahead ? next_s - next_o < 2 : fill)) {
          ok = ok && ptx::mbar_wait(smem_addr(&full[s_stage]), s_phase, &g_latent_status, (7 << 8) | 2);
          __syncwarp();
          ptx::tc_fence_after();
          uint32_t aq = static_cast<uint32_t>(dq), bk = static_cast<uint32_t>(dk) + s_stage * stage_step;
          const uint32_t d = tmem_s + (next_s & 1) * kPage;
#pragma unroll 1
          for (int b = 0; b < p.boxes; ++b) {  // (columns beyond the row are zero in both operands)
#pragma unroll
            for (int j = 0; j < 4; ++j) mma_f16_ss(lead, d, aq + 2 * j, k_hi, bk + 2 * j, k_hi, id_s, (b | j) > 0 ? 1u : 0u);
            aq += NR * 128 >> 4;
            bk += kBoxBytes >> 4;
          }
          if (lead) ptx::tc_commit(smem_addr(&bar_s[next_s & 1]));
          __syncwarp();
          if (++s_stage == p.stages) { s_stage = 0; s_phase ^= 1; }
          ++next_s;
          fill = next_s - next_o < 2;
          continue;
        }
        ok = ok && ptx::mbar_wait(smem_addr(&bar_p[next_o & 1]), (next_o >> 1) & 1, &g_latent_status, (7 << 8) | 4);
        __syncwarp();
        ptx::tc_fence_after();
        uint32_t av = static_cast<uint32_t>(dv) + o_stage * stage_step;
        const uint32_t pb = static_cast<uint32_t>(dp) + (p.p_in_page ? o_stage * stage_step : (next_o & 1) * (NR * 128 >> 4));
#pragma unroll 1
        for (int m = 0; m < p.blocks; ++m) {
#pragma unroll
          for (int j = 0; j < 4; ++j)        // 16 keys
            mma_f16_ss(lead, tmem + m * NR, av + j * (2048 >> 4), v_hi, pb + 2 * j, k_hi, id_o, next_o > 0 || j > 0 ? 1u : 0u);
          av += 2 * kBoxBytes >> 4;
        }
        if (lead) {
          ptx::tc_commit(smem_addr(&empty[o_stage]));
          ptx::tc_commit(smem_addr(bar_o));
        }
        __syncwarp();
        if (++o_stage == p.stages) o_stage = 0;
        ++next_o;
        fill = next_o == next_s;
      }
      if (lead) ptx::tc_commit(smem_addr(bar_done));
    }
    __syncwarp();
  } else {
    // ------- softmax: rows r0 = 16 (warp % 4) + lane / 4 and r0 + 8, keys 32 (warp / 4) + 8 j + 2 (lane % 4) + {0, 1} -------
    const int quarter = warp & 3, half = warp >> 2;
    const bool band = quarter * 16 < NR;     // (with a 32-row tile half of the warps only rescale and store)
    const int r0 = quarter * 16 + (lane >> 2);
    float m_ref[2], l_run[2];
    int row_pos[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = r0 + 8 * e;
      const bool real = band && r < used;
      row_pos[e] = real ? pos0 + r / nheads : -1;
      m_ref[e] = (real && split == 0) ? p.sink[head0 + r % nheads] * kLog2e : -1e30f;
      l_run[e] = (real && split == 0 && half == 0 && (lane & 3) == 0) ? 1.f : 0.f;
    }
    const float qscale = a.scale * kLog2e;
    const uint32_t lane_addr = static_cast<uint32_t>(quarter * 32) << 16;
    for (int it = 0; it < npages; ++it) {
      uint8_t* p_tile = p.p_in_page ? s_kv + stage * page_bytes + 2 * p.blocks * kBoxBytes : s_p + (it & 1) * NR * 128;
      ok = ok && ptx::mbar_wait(smem_addr(&bar_s[it & 1]), (it >> 1) & 1, &g_latent_status, (7 << 8) | 5);
      __syncwarp();
      ptx::tc_fence_after();
      float s[16], alpha[2] = {1.f, 1.f};
      bool grown = false;
      const int base = (pg_begin + it) * kPage;
      if (band) {
        tmem_ld_rows16(tmem_s + (it & 1) * kPage + half * 32 + lane_addr, s);
        float mx[2] = {-1e30f, -1e30f};
        if (base + kPage - 1 <= pos0 && base > pos_last - a.window) {      // the whole page is seen by every row
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            s[i] *= qscale;
            mx[(i >> 1) & 1] = fmaxf(mx[(i >> 1) & 1], s[i]);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const int key = base + half * 32 + (i >> 2) * 8 + (lane & 3) * 2 + (i & 1), rp = row_pos[(i >> 1) & 1];
            s[i] = (key <= rp && key > rp - a.window) ? s[i] * qscale : -INFINITY;
            mx[(i >> 1) & 1] = fmaxf(mx[(i >> 1) & 1], s[i]);
          }
        }
#pragma unroll
        for (int off = 1; off < 4; off <<= 1)
#pragma unroll
          for (int e = 0; e < 2; ++e) mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], off));
        if ((lane & 3) == 0) {
          s_max[((it & 1) * 2 + half) * NR + r0] = mx[0];
          s_max[((it & 1) * 2 + half) * NR + r0 + 8] = mx[1];
        }
        // (this half's keys decide for the row as soon as they exceed the bound)
        grown = it > 0 && ((row_pos[0] >= 0 && mx[0] > m_ref[0] + kStale) || (row_pos[1] >= 0 && mx[1] > m_ref[1] + kStale));
      }
      const int tail = pos_last + 1 - base;
      if (tail < kPage) {                    // rows behind the last token may hold anything: zero, so that 0 * row stays 0
        for (int i = threadIdx.x; i < (kPage - tail) * p.boxes * 8; i += kSoftThreads) {
          const int r = tail + i / (p.boxes * 8), c = i % (p.boxes * 8);
          *reinterpret_cast<uint4*>(s_kv + stage * page_bytes + (c >> 3) * kBoxBytes + r * 128 + (c & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      }
      if (++stage == p.stages) stage = 0;
      const bool rescale = any_softmax(grown);       // (also publishes s_max)
      if (band) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float mx = fmaxf(s_max[(it & 1) * 2 * NR + r0 + 8 * e], s_max[((it & 1) * 2 + 1) * NR + r0 + 8 * e]);
          if (row_pos[e] >= 0 && mx > m_ref[e] + (it == 0 ? 0.f : kStale)) {
            alpha[e] = ex2(m_ref[e] - mx);
            m_ref[e] = mx;
          }
        }
      }
      if (rescale) {                         // rare: bring O^T to the new references
        if (band && half == 0 && (lane & 3) == 0) {
          s_alpha[r0] = alpha[0];
          s_alpha[r0 + 8] = alpha[1];
        }
        ok = ok && ptx::mbar_wait(smem_addr(bar_o), (it - 1) & 1, &g_latent_status, (7 << 8) | 6);     // the page before is in (the one before that is: this page's scores follow it)
        __syncwarp();
        ptx::tc_fence_after();
        sync_softmax();
        for (int c = half * 16; c < p.blocks * NR; c += 32) {
          float o[16];
          tmem_ld_x16(tmem + lane_addr + c, o);
#pragma unroll
          for (int j = 0; j < 16; ++j) o[j] *= s_alpha[(c + j) % NR];
          tmem_st_x16(tmem + lane_addr + c, o);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        sync_softmax();                      // s_alpha may be written again
      }
      if (band) {
#pragma unroll
        for (int e = 0; e < 2; ++e) l_run[e] *= alpha[e];
        uint8_t* dst = p_tile + r0 * 128 + (lane & 3) * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            s[4 * j + e] = row_pos[e >> 1] >= 0 ? ex2(s[4 * j + e] - m_ref[e >> 1]) : 0.f;
            l_run[e >> 1] += s[4 * j + e];
          }
          const int chunk = ((half * 4 + j) ^ (lane >> 2)) << 4;           // (both rows are lane / 4 modulo 8)
          *reinterpret_cast<uint32_t*>(dst + chunk) = pack_bf16(s[4 * j], s[4 * j + 1]);
          *reinterpret_cast<uint32_t*>(dst + 8 * 128 + chunk) = pack_bf16(s[4 * j + 2], s[4 * j + 3]);
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");       // the tensor core reads what was just written
      }
      ptx::tc_fence_before();
      ptx::mbar_arrive(smem_addr(&bar_p[it & 1]));
    }
    // references and denominators (s_max: the two key halves' sums)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 1);
      l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 2);
    }
    sync_softmax();
    if (band && (lane & 3) == 0) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (half == 0) s_ml[r0 + 8 * e] = m_ref[e];
        s_max[half * NR + r0 + 8 * e] = l_run[e];
      }
    }
    // (not by bar_o: with scores issued ahead the page before the last may still be in the works, and its phase would alias)
    if (npages > 0) ok = ok && ptx::mbar_wait(smem_addr(bar_done), 0, &g_latent_status, (7 << 8) | 7);
    __syncwarp();
    ptx::tc_fence_after();
    sync_softmax();                          // every page has been read: the ring is free
    if (threadIdx.x < NR) {
      const float l = s_max[threadIdx.x] + s_max[NR + threadIdx.x];
      s_ml[NR + threadIdx.x] = l;
      s_alpha[threadIdx.x] = 1.f / l;
    }
    sync_softmax();
    // O^T (lane = latent column of the block, tensor-memory column = tile row) turns in shared memory: as finished bf16
    // rows, or as float parts of a split tile
    __nv_bfloat16* s_out = reinterpret_cast<__nv_bfloat16*>(smem);
    float* s_o = reinterpret_cast<float*>(smem);
    const int bpitch = a.kv_rank + 8, opitch = a.kv_rank + 4;
    for (int u = half; u < p.blocks * (NR / 16); u += 2) {
      const int m = u / (NR / 16), c = (u % (NR / 16)) * 16;
      if (c >= used) continue;
      const int col = m * 128 + quarter * 32 + lane;
      float o[16];
      if (npages > 0) {
        tmem_ld_x16(tmem + lane_addr + m * NR + c, o);
      } else {
#pragma unroll
        for (int j = 0; j < 16; ++j) o[j] = 0.f;
      }
      if (col < a.kv_rank) {
        if (p.splits == 1) {
#pragma unroll
          for (int j = 0; j < 16; ++j) s_out[(c + j) * bpitch + col] = __float2bfloat16_rn(o[j] * s_alpha[c + j]);
        } else {
#pragma unroll
          for (int j = 0; j < 16; ++j) s_o[(c + j) * opitch + col] = o[j];
        }
      }
      __syncwarp();
    }
    if (p.splits == 1) {
      sync_softmax();
      const int pieces = a.kv_rank / 8;
      __nv_bfloat16* dst = p.out + (static_cast<size_t>(row0) * a.heads + head0) * a.kv_rank;      // neighbouring rows
      for (int i = threadIdx.x; i < used * pieces; i += kSoftThreads) {
        const int r = i / pieces, c = i % pieces;
        *reinterpret_cast<uint4*>(dst + static_cast<size_t>(i) * 8) = *reinterpret_cast<const uint4*>(s_out + r * bpitch + c * 8);
      }
    }
  }
  if (p.splits > 1) {
    // The cluster's CTAs share one tile. CTA d finishes rows d * share ..; every CTA sends it those rows of its part with one
    // bulk copy, so that the sums read local memory. Parts are added in rank order.
    const int opitch = a.kv_rank + 4, share = (used + p.splits - 1) / p.splits;
    const int mine = min(max(used - split * share, 0), share);
    float* s_o = reinterpret_cast<float*>(smem);
    float* s_in = s_o + NR * opitch;                            // [splits][share][opitch]
    const uint32_t bar_in = smem_addr(bar_q);                   // its second phase
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // this CTA's part, before the copy engine reads it
    if (threadIdx.x == 0) ptx::mbar_expect_tx(bar_in, p.splits * mine * opitch * 4);
    __syncwarp();
    cluster_sync_all();                    // every ring is drained, every barrier is armed
    if (threadIdx.x < p.splits) {
      const int d = (split + threadIdx.x) % p.splits, rows = min(max(used - d * share, 0), share);
      if (rows > 0)
        ptx::bulk_copy_to_rank(smem_addr(s_in + split * share * opitch), smem_addr(s_o + d * share * opitch), rows * opitch * 4, bar_in, d);
    }
    // references and denominators of my rows in every part
    for (int i = threadIdx.x; i < mine * p.splits; i += kThreads) {
      const int k = i / p.splits, src = i - k * p.splits;
      s_w[(k * kMaxSplits + src) * 2] = ld_peer_f32(smem_addr(s_ml + split * share + k), src);
      s_w[(k * kMaxSplits + src) * 2 + 1] = ld_peer_f32(smem_addr(s_ml + NR + split * share + k), src);
    }
    __syncthreads();
    // (phase 0 is over when this CTA loaded its queries, else it is the current one)
    ok = ptx::mbar_wait(bar_in, npages > 0 ? 1 : 0, &g_latent_status, (7 << 8) | 10) && ok;
    const int pieces = a.kv_rank / 8;
#pragma unroll 1
    for (int i = threadIdx.x; i < mine * pieces; i += kThreads) {
      const int k = i / pieces, c = (i - k * pieces) * 8;
      const float* ml = s_w + k * kMaxSplits * 2;
      float top = ml[0], sum = 0.f, v[8] = {};
#pragma unroll 1
      for (int part = 1; part < p.splits; ++part) top = fmaxf(top, ml[2 * part]);
#pragma unroll 1
      for (int part = 0; part < p.splits; ++part) {
        const float w = ex2(ml[2 * part] - top);
        sum = fmaf(ml[2 * part + 1], w, sum);
        const float4* src = reinterpret_cast<const float4*>(s_in + (part * share + k) * opitch + c);
        const float4 x = src[0], y = src[1];
        v[0] = fmaf(x.x, w, v[0]); v[1] = fmaf(x.y, w, v[1]); v[2] = fmaf(x.z, w, v[2]); v[3] = fmaf(x.w, w, v[3]);
        v[4] = fmaf(y.x, w, v[4]); v[5] = fmaf(y.y, w, v[5]); v[6] = fmaf(y.z, w, v[6]); v[7] = fmaf(y.w, w, v[7]);
      }
      const float inv = 1.f / sum;
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= inv;
      VecIO<__nv_bfloat16, 8>::st(p.out + (static_cast<size_t>(row0) * a.heads + head0 + split * share + k) * a.kv_rank + c, v);
    }
    __syncwarp();
    cluster_sync_all();                    // nobody leaves while its part is being read
  }
  ptx::tc_fence_before();
  __syncthreads();
  if (warp == 8) {
    ptx::tc_fence_after();
    ptx::tc_dealloc(tmem, p.tmem_cols);
  }
}

constexpr size_t kSmemLimit = 227 * 1024;
int row_boxes(int width) { return (width + 63) / 64; }
// Shared memory beside the ring, and the pages that fit (at least two).
size_t fast_fixed_smem(int nr, int boxes, int p_in_page) {
  // (the score MMAs read 64 query rows: behind a 32-row tile's last box lies memory of this block)
  const size_t behind = p_in_page && nr == 32 ? 4096 : 0;
  return 1024 + behind + static_cast<size_t>(boxes + (p_in_page ? 0 : 2)) * nr * 128 + nr * 7 * 4 + (2 * kMaxStages + 8) * 8 + 16;
}
int latent_blocks(int kv_rank) { return (kv_rank + 127) / 128; }
int prob_in_page(int kv_rank, int width) { return row_boxes(width) > 2 * latent_blocks(kv_rank) ? 1 : 0; }
int fast_stages(int nr, int kv_rank, int width) {
  const int boxes = row_boxes(width);
  const size_t page = static_cast<size_t>(boxes) * kBoxBytes, fixed = fast_fixed_smem(nr, boxes, prob_in_page(kv_rank, width));
  int s = fixed > kSmemLimit ? 0 : static_cast<int>((kSmemLimit - fixed) / page);
  if (s > kMaxStages) s = kMaxStages;
  return s >= 2 ? s : 0;
}
int tile_rows(int kv_rank, int width) { return fast_stages(64, kv_rank, width) > 0 ? 64 : 32; }
int head_groups(int heads, int rows) { return (heads + rows - 1) / rows; }

bool encode_rows(CUtensorMap* map, const void* base, uint64_t width, uint64_t rows, uint32_t box_rows) {
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

template <int NR>
int launch_fast(FastParams p, const void* q, dim3 grid, cudaStream_t st) {
  const int width = p.a.kv_rank + p.a.rot_dim;
  p.stages = fast_stages(NR, p.a.kv_rank, width);
  if (p.stages == 0) return CACHEIR_B200_EUNSUPPORTED;
  p.boxes = row_boxes(width);
  p.blocks = latent_blocks(p.a.kv_rank);
  p.ahead = p.stages >= 3 ? 1 : 0;
  p.p_in_page = prob_in_page(p.a.kv_rank, width);
  const int cols = p.blocks * NR + 2 * kPage;
  p.tmem_cols = cols <= 256 ? 256 : 512;
  size_t smem = fast_fixed_smem(NR, p.boxes, p.p_in_page) + static_cast<size_t>(p.stages) * p.boxes * kBoxBytes;
  // the combine's tile and what the peers send lie over the ring
  const size_t combine = static_cast<size_t>(NR + (NR + p.splits - 1) / p.splits * p.splits) * (p.a.kv_rank + 4) * 4;
  if (p.splits > 1 && combine > static_cast<size_t>(p.stages) * p.boxes * kBoxBytes) return CACHEIR_B200_EUNSUPPORTED;
  // No more CTAs on an SM than its tensor memory serves: one that waited for an allocation could hold up its cluster.
  const size_t least = kSmemLimit / (512 / p.tmem_cols + 1) + 1024;
  if (smem < least) smem = least;
  CUtensorMap tkv, tq;
  if (!encode_rows(&tkv, p.a.pool, width, static_cast<uint64_t>(p.a.num_slots) * kPage, kPage) ||
      !encode_rows(&tq, q, width, static_cast<uint64_t>(p.a.rows) * p.a.heads, NR))
    return CACHEIR_B200_EUNSUPPORTED;
  auto kern = latent_attention_kernel<NR>;
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
  e = cudaLaunchKernelEx(&cfg, kern, tkv, tq, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  return launch_status();
}

bool latent_args_ok(const cacheir_b200_latent_args& a) {
  return a.positions && a.row_seg && a.page_table && a.pool && a.segments > 0 && a.max_pages > 0 && a.page_size > 0 && a.num_slots > 0 &&
         a.heads > 0 && a.dim > 0 && a.rot_dim >= 0 && a.vdim > 0 && a.kv_rank > 0 && a.window > 0 && a.heads <= 65535;
}

}  // namespace

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
  return dtype == CACHEIR_B200_BF16 && page_size == kPage && kv_rank >= 8 && kv_rank % 8 == 0 && kv_rank <= 512 && rot_dim >= 0 &&
         rot_dim % 8 == 0 && fast_stages(32, kv_rank, kv_rank + rot_dim) > 0 ? 1 : 0;
}

extern "C" int cacheir_b200_latent_attention_splits(int rows, int heads, int window, int max_pages, int page_size) {
  if (rows <= 0 || heads <= 0 || page_size <= 0) return 1;
  const int units = rows * head_groups(heads, 64);
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
  p.sink = sink;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.splits = splits;
  int rows = splits > 1 ? 32 : tile_rows(a.kv_rank, a.kv_rank + a.rot_dim);      // (a split 64-row tile would not fit its combine)
  const int groups = head_groups(a.heads, rows);
  p.heads_per_cta = (a.heads + groups - 1) / groups;
  if (decode && p.heads_per_cta <= 32) rows = 32;
  p.tokens_per_tile = decode ? 1 : rows / p.heads_per_cta;
  const int items = decode ? a.rows : ragged_items(a.rows, a.segments, p.tokens_per_tile);
  const dim3 grid(items, groups, splits);
  return rows == 64 ? launch_fast<64>(p, q, grid, as_stream(stream)) : launch_fast<32>(p, q, grid, as_stream(stream));
}

extern "C" int cacheir_b200_hybrid_device_status(int reset) { return device_status_word(g_latent_status, reset != 0); }
