// Tied attention (values are the projected keys) over a paged cache, sm_100a: preparation, the plain form, and decoding.
//
// prepare   one warp per head: root mean square, rotation; queries go to a buffer, keys to their cache row.
// simple    any extents, float32 arithmetic: one CTA per (row, head).
// step      one CTA per (sequence, key/value head, split). Pages of 64 cached rows land in a ring as TMA boxes of 64 columns;
//           a row is read once and serves as key (columns from rot_dims on, times its reciprocal root mean square) and as
//           value (the first dim columns). Four warps take 16 rows of a page each with warp MMAs, the heads of the group
//           being the 16-row operand; they meet once per CTA, and splits meet in distributed shared memory.
#include "tied_attention.cuh"

namespace cb200 {
namespace {

__device__ int g_tied_status = 0;

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
tied_prepare_kernel(const cacheir_b200_tied_args a, const T* __restrict__ q, long long q_stride, const T* __restrict__ k, long long k_stride,
                    float eps, const float2* __restrict__ table, int table_positions, T* __restrict__ q_out) {
  const int row = blockIdx.x, lane = threadIdx.x & 31;
  const int unit = blockIdx.y * 8 + (threadIdx.x >> 5);      // query heads, then key heads
  const int seg = a.row_seg[row], pos = a.positions[row];
  if (seg < 0 || unit >= a.heads + a.kv_heads || pos < 0 || pos >= table_positions || pos / a.page_size >= a.max_pages) return;
  const bool key = unit >= a.heads;
  const int head = key ? unit - a.heads : unit;
  const T* src = key ? k + static_cast<size_t>(row) * k_stride + static_cast<size_t>(head) * a.dim
                     : q + static_cast<size_t>(row) * q_stride + static_cast<size_t>(head) * a.dim;
  const int half = a.rot_dims / 2, lead = tied_lead(a.rot_dims);
  T *plain, *turned;            // where entry c goes as it is, and rotated entry c
  float* inv_out = nullptr;
  if (key) {
    const int slot = a.page_table[static_cast<size_t>(seg) * a.max_pages + pos / a.page_size];
    if (slot < 0 || slot >= a.num_slots) return;
    const size_t at = (static_cast<size_t>(slot) * a.kv_heads + head) * a.page_size + pos % a.page_size;
    plain = static_cast<T*>(a.pool) + at * (a.dim + a.rot_dims);
    turned = plain + a.dim;
    inv_out = a.inv_rms + at;
  } else {
    plain = q_out + (static_cast<size_t>(row) * a.heads + head) * (a.dim + a.rot_dims - lead) - lead;
    turned = plain + a.dim;
  }
  float ss = 0.f;
  for (int c = lane * VEC; c < a.dim; c += 32 * VEC) {
    float v[VEC];
    load_vec<T, VEC>(src + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(a.dim) + eps);
  const float by = key ? 1.f : inv;        // keys keep their length: the values are the same rows
  const float2* cs = table + static_cast<size_t>(pos) * half;
  for (int c = lane * VEC; c < a.dim; c += 32 * VEC) {
    float v[VEC];
    load_vec<T, VEC>(src + c, v);
    if (c < a.rot_dims) {
      const bool low = c < half;
      float other[VEC], r[VEC];
      load_vec<T, VEC>(src + (low ? c + half : c - half), other);
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const float2 t = cs[(low ? c : c - half) + i];
        r[i] = (low ? v[i] * t.x - other[i] * t.y : v[i] * t.x + other[i] * t.y) * by;
      }
      store_vec<T, VEC>(turned + c, r);
      if (!key) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = 0.f;
      }
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] *= by;
    }
    if (key || c >= lead) store_vec<T, VEC>(plain + c, v);
  }
  if (key && lane == 0) *inv_out = inv;
}

// ---- plain form ------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
tied_simple_kernel(const cacheir_b200_tied_args a, const T* __restrict__ q, const T* __restrict__ gate, long long gate_stride,
                   T* __restrict__ out) {
  extern __shared__ float sm[];
  __shared__ float scratch[32];
  const int lead = tied_lead(a.rot_dims), width = a.dim + a.rot_dims, qw = width - lead;
  float* sq = sm;                     // [qw]
  float* so = sq + qw;                // [dim]
  float* sp = so + a.dim;             // [128]
  const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int seg = a.row_seg[row];
  if (seg < 0) return;
  const int pos = a.positions[row], kvh = h / (a.heads / a.kv_heads);
  for (int c = tid; c < qw; c += 128) sq[c] = Elem<T>::ld(q + (static_cast<size_t>(row) * a.heads + h) * qw + c);
  for (int c = tid; c < a.dim; c += 128) so[c] = 0.f;
  float m = a.sink ? a.sink[h] : -1e30f, l = a.sink ? 1.f : 0.f;
  __syncthreads();
  auto cached = [&](int j) {          // index of position j's row among all rows of the pool
    return (static_cast<size_t>(tied_slot(a, seg, j / a.page_size)) * a.kv_heads + kvh) * a.page_size + j % a.page_size;
  };
  auto attend = [&](int begin, int end) {
    for (int k0 = begin; k0 < end; k0 += 128) {
      const int j = k0 + tid;
      float s = -INFINITY;
      if (j < end) {
        const size_t at = cached(j);
        const T* kr = static_cast<const T*>(a.pool) + at * width + lead;
        float dot = 0.f;
        for (int c = 0; c < qw; ++c) dot = fmaf(sq[c], Elem<T>::ld(kr + c), dot);
        s = dot * a.inv_rms[at] * a.scale;
        if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
      }
      const float wm = warp_max(s);
      if ((tid & 31) == 0) scratch[tid >> 5] = wm;
      __syncthreads();
      const float m_new = fmaxf(m, fmaxf(fmaxf(scratch[0], scratch[1]), fmaxf(scratch[2], scratch[3])));
      const float p = j < end ? expf(s - m_new) : 0.f;
      sp[tid] = p;
      const float alpha = expf(m - m_new);
      l = l * alpha + block_sum_all(p, scratch);      // (its barriers also publish sp)
      m = m_new;
      const int n = min(128, end - k0);
      for (int c = tid; c < a.dim; c += 128) {
        float acc = so[c] * alpha;
        for (int i = 0; i < n; ++i) acc = fmaf(sp[i], Elem<T>::ld(static_cast<const T*>(a.pool) + cached(k0 + i) * width + c), acc);
        so[c] = acc;
      }
      __syncthreads();
    }
  };
  const int lo = max(0, pos - a.window + 1);
  attend(0, min(a.keep_first, lo));
  attend(lo, pos + 1);
  const float inv = 1.f / l;
  for (int c = tid; c < a.dim; c += 128) {
    float o = so[c] * inv;
    if (gate) o *= sigmoid_exact(Elem<T>::ld(gate + static_cast<size_t>(row) * gate_stride + static_cast<size_t>(h) * a.dim + c));
    Elem<T>::st(out + (static_cast<size_t>(row) * a.heads + h) * a.dim + c, o);
  }
}

// ---- decoding --------------------------------------------------------------------------------------------------------
constexpr int kWarps = 4;                        // consumer warps; one more copies
constexpr int kStepThreads = (kWarps + 1) * 32;
constexpr int kMaxStages = 6;
constexpr int kMaxSplits = 8;                    // CTAs of a cluster

struct StepParams {
  cacheir_b200_tied_args a;
  const __nv_bfloat16* q;
  const __nv_bfloat16* gate;
  long long gate_stride;
  __nv_bfloat16* out;
  TiedScore score;
  int subs, heads_per_cta, splits, boxes, stages;
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

// DB: 64-column boxes of the values; kSteps: 32-column pieces of a row that queries meet
template <int DB, int kSteps>
__global__ void __launch_bounds__(kStepThreads, DB <= 2 ? 2 : 1)
tied_step_kernel(const __grid_constant__ CUtensorMap tmap, const StepParams p) {
  constexpr int kTiles = DB * 8;                 // 8-column tiles of the output
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const cacheir_b200_tied_args& a = p.a;
  const int page_bytes = p.boxes * kTiedBox;
  float* s_inv = reinterpret_cast<float*>(smem + p.stages * page_bytes);      // [stages][64]
  uint64_t* full = reinterpret_cast<uint64_t*>(s_inv + p.stages * kTiedPage);
  uint64_t* empty = full + kMaxStages;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, seg = blockIdx.z;          // (the cluster spans the whole x extent)
  const int kvh = blockIdx.y / p.subs, sub = blockIdx.y % p.subs;
  const int group = a.heads / a.kv_heads;
  const int head0 = kvh * group + sub * p.heads_per_cta;
  const int nheads = min(p.heads_per_cta, group - sub * p.heads_per_cta);
  if (a.row_seg[seg] < 0) return;                          // (a padding row: the whole cluster leaves)
  const int pos = a.positions[seg];
  const TiedPages pages(a, pos, pos);
  const int begin = pages.total * split / p.splits, n = pages.total * (split + 1) / p.splits - begin;

  if (threadIdx.x == 0) {
    for (int s = 0; s < p.stages; ++s) { ptx::mbar_init(smem_addr(&full[s]), 1); ptx::mbar_init(smem_addr(&empty[s]), kWarps); }
    ptx::mbar_fence_init();
  }
  __syncthreads();

  const int g = lane >> 2, t4 = lane & 3;
  float m_run[2] = {-1e30f, -1e30f}, l_run[2] = {0.f, 0.f};
  float o[kTiles][4];
#pragma unroll
  for (int i = 0; i < kTiles; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;

  if (warp == kWarps) {
    // ---------------- copies ----------------
    int slots = 0, issued = 0;
    for (int it = 0; it < n; ++it) {
      if (it % 32 == 0) slots = it + lane < n ? tied_slot(a, seg, pages.page(begin + it + lane)) : 0;
      const int slot = __shfl_sync(0xffffffffu, slots, it % 32);
      bool ok = true;
      if (lane == 0) {
        const int s = it % p.stages;
        if (it >= p.stages) ok = ptx::mbar_wait(smem_addr(&empty[s]), ((it / p.stages) & 1) ^ 1, &g_tied_status, (8 << 8) | 1);
        if (ok) {
          const uint32_t bar = smem_addr(&full[s]);
          const int unit = slot * a.kv_heads + kvh;
          ptx::mbar_expect_tx(bar, page_bytes + kTiedPage * 4);
          for (int b = 0; b < p.boxes; ++b) ptx::tma_load_2d(smem_addr(smem + s * page_bytes + b * kTiedBox), &tmap, bar, b * 64, unit * kTiedPage);
          ptx::bulk_load(smem_addr(s_inv + s * kTiedPage), a.inv_rms + static_cast<size_t>(unit) * kTiedPage, kTiedPage * 4, bar);
          issued = it + 1;
        }
      }
      if (!__shfl_sync(0xffffffffu, ok ? 1 : 0, 0)) break;
    }
    if (lane == 0 && issued < n)        // a wait gave up: nothing may still be on its way when the block ends
      for (int it = max(0, issued - p.stages); it < issued; ++it)
        ptx::mbar_wait(smem_addr(&full[it % p.stages]), (it / p.stages) & 1, &g_tied_status, (8 << 8) | 2);
  } else {
    // ---------------- four warps, 16 keys of every page each ----------------
    const int width = a.dim + a.rot_dims, lead = tied_lead(a.rot_dims), qw = width - lead;
    const int k_first = a.rot_dims / 32, last_piece = p.boxes * 2 - 1;      // (a piece behind the row meets zero queries: any data will do)
    uint32_t qa[kSteps][2][4];
    const __nv_bfloat16* qb = p.q + (static_cast<size_t>(seg) * a.heads + head0) * qw - lead;
#pragma unroll
    for (int k = 0; k < kSteps; ++k)
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          const int head = g + (r & 1) * 8, col = (k_first + k) * 32 + half * 16 + 2 * t4 + (r >> 1) * 8;
          qa[k][half][r] = (head < nheads && col < width) ? *reinterpret_cast<const uint32_t*>(qb + static_cast<size_t>(head) * qw + col) : 0u;
        }
    const uint32_t lrow = lane & 7, lmat = lane >> 3;
    bool ok = true;
    for (int it = 0; it < n; ++it) {
      const int s = it % p.stages;
      ok = ptx::mbar_wait(smem_addr(&full[s]), (it / p.stages) & 1, &g_tied_status, (8 << 8) | 3);
      if (!__all_sync(0xffffffffu, ok)) break;
      const int base = pages.page(begin + it) * kTiedPage + warp * 16;       // position of this warp's first key
      uint8_t* page = smem + s * page_bytes;
      if (base + 15 > pos) {               // rows behind the last token may hold anything: zero, so that 0 * row stays 0
        const int valid = max(0, pos + 1 - base);
        for (int i = lane; i < (16 - valid) * p.boxes * 8; i += 32) {
          const int r = warp * 16 + valid + i / (p.boxes * 8), c = i % (p.boxes * 8);
          *reinterpret_cast<uint4*>(page + (c >> 3) * kTiedBox + r * 128 + (c & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
        __syncwarp();
      }
      const uint32_t rows = smem_addr(page) + warp * 16 * 128;
      // scores: both 8-key tiles side by side, even and odd pieces in sums of their own (shorter dependent chains)
      float sc[2][4], sd[2][4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nt][e] = sd[nt][e] = 0.f;
#pragma unroll
      for (int k = 0; k < kSteps; ++k) {
        const uint32_t c = 4 * min(k_first + k, last_piece) + lmat;        // 16-byte piece of the row
        const uint32_t at = rows + (c >> 3) * kTiedBox + lrow * 128 + (((c & 7) ^ lrow) << 4);
        uint32_t kb[2][4];
        ldsm_x4(at, kb[0]);
        ldsm_x4(at + 8 * 128, kb[1]);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_bf16(sc[nt], qa[k][0], kb[nt][0], kb[nt][1]);
          mma_bf16(sd[nt], qa[k][1], kb[nt][2], kb[nt][3]);
        }
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nt][e] += sd[nt][e];
      float pmax[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        const float2 inv = *reinterpret_cast<const float2*>(s_inv + s * kTiedPage + warp * 16 + nt * 8 + 2 * t4);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = base + nt * 8 + 2 * t4 + (e & 1);
          const bool seen = key <= pos && (key > pos - a.window || key < a.keep_first);
          const float v = seen ? p.score(sc[nt][e] * ((e & 1) ? inv.y : inv.x)) : -INFINITY;
          sc[nt][e] = v;
          pmax[e >> 1] = fmaxf(pmax[e >> 1], v);
        }
      }
      float corr[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        pmax[r] = fmaxf(pmax[r], __shfl_xor_sync(0xffffffffu, pmax[r], 1));
        pmax[r] = fmaxf(pmax[r], __shfl_xor_sync(0xffffffffu, pmax[r], 2));
        const float m_new = fmaxf(m_run[r], pmax[r]);
        corr[r] = tied_ex2(m_run[r] - m_new);
        m_run[r] = m_new;
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nt][e] = tied_ex2(sc[nt][e] - m_run[e >> 1]);
#pragma unroll
      for (int r = 0; r < 2; ++r) l_run[r] = l_run[r] * corr[r] + (sc[0][2 * r] + sc[0][2 * r + 1] + sc[1][2 * r] + sc[1][2 * r + 1]);
      const uint32_t pa[4] = {pack_bf16(sc[0][0], sc[0][1]), pack_bf16(sc[0][2], sc[0][3]), pack_bf16(sc[1][0], sc[1][1]),
                              pack_bf16(sc[1][2], sc[1][3])};
      if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < kTiles; ++i) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
      }
#pragma unroll
      for (int j = 0; j < kTiles / 2; ++j) {
        const uint32_t token = (lmat & 1) * 8 + lrow, c = 2 * j + (lmat >> 1);       // (columns behind dim are computed and not kept)
        uint32_t vb[4];
        ldsm_x4_t(rows + (c >> 3) * kTiedBox + token * 128 + (((c & 7) ^ lrow) << 4), vb);
        mma_bf16(o[2 * j], pa, vb[0], vb[1]);
        mma_bf16(o[2 * j + 1], pa, vb[2], vb[3]);
      }
      __syncwarp();
      if (lane == 0) ptx::mbar_arrive(smem_addr(&empty[s]));
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
      l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    }
  }

  // ---------------- the warps meet over the drained ring, then the cluster's CTAs ----------------
  __syncthreads();
  float* s_m = reinterpret_cast<float*>(smem);                  // [warps][16]
  float* s_l = s_m + kWarps * 16;                               // [warps][16]
  float* s_o = s_l + kWarps * 16;                               // [warps][16][dim]
  if (warp < kWarps) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = g + r * 8;
      if (t4 == 0) { s_m[warp * 16 + row] = m_run[r]; s_l[warp * 16 + row] = l_run[r]; }
#pragma unroll
      for (int i = 0; i < kTiles; ++i)
        if (i * 8 < a.dim)
          *reinterpret_cast<float2*>(s_o + (warp * 16 + row) * a.dim + i * 8 + 2 * t4) = make_float2(o[i][2 * r], o[i][2 * r + 1]);
    }
  }
  __syncthreads();
  auto finish = [&](int row, int d, float m, float l, float acc) {           // the sink joins here
    const int head = head0 + row;
    const float sink = a.sink ? a.sink[head] * kLog2e : -1e30f;
    const float top = fmaxf(m, sink), by = tied_ex2(m - top);
    float y = acc * by / (l * by + (a.sink ? tied_ex2(sink - top) : 0.f));
    const size_t col = static_cast<size_t>(head) * a.dim + d;
    if (p.gate) y *= sigmoid_exact(__bfloat162float(p.gate[static_cast<size_t>(seg) * p.gate_stride + col]));
    p.out[static_cast<size_t>(seg) * a.heads * a.dim + col] = __float2bfloat16_rn(y);
  };
  auto meet = [&](int row, int d, float& m, float& l, float& acc) {          // this CTA's four parts
    m = s_m[row];
#pragma unroll
    for (int w = 1; w < kWarps; ++w) m = fmaxf(m, s_m[w * 16 + row]);
    l = acc = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float by = tied_ex2(s_m[w * 16 + row] - m);
      l = fmaf(s_l[w * 16 + row], by, l);
      acc = fmaf(s_o[(w * 16 + row) * a.dim + d], by, acc);
    }
  };
  if (p.splits == 1) {
    for (int i = threadIdx.x; i < nheads * a.dim; i += kStepThreads) {
      float m, l, acc;
      meet(i / a.dim, i % a.dim, m, l, acc);
      finish(i / a.dim, i % a.dim, m, l, acc);
    }
    return;
  }
  float* s_part = s_o + kWarps * 16 * a.dim;                    // [16] m, [16] l of the whole CTA
  for (int i = threadIdx.x; i < nheads * a.dim; i += kStepThreads) {
    const int row = i / a.dim, d = i % a.dim;
    float m, l, acc;
    meet(row, d, m, l, acc);
    s_o[row * a.dim + d] = acc;                                 // (this thread alone reads and writes the element)
    if (d == 0) { s_part[row] = m; s_part[16 + row] = l; }
  }
  __syncwarp();
  cluster_sync_all();
  for (int i = split * kStepThreads + threadIdx.x; i < nheads * a.dim; i += p.splits * kStepThreads) {
    const int row = i / a.dim, d = i % a.dim;
    float ms[kMaxSplits], m = -1e30f, l = 0.f, acc = 0.f;
#pragma unroll
    for (int r = 0; r < kMaxSplits; ++r) {
      ms[r] = r < p.splits ? ld_peer_f32(s_part + row, r) : -1e30f;
      m = fmaxf(m, ms[r]);
    }
#pragma unroll
    for (int r = 0; r < kMaxSplits; ++r)
      if (r < p.splits) {
        const float by = tied_ex2(ms[r] - m);
        l = fmaf(ld_peer_f32(s_part + 16 + row, r), by, l);
        acc = fmaf(ld_peer_f32(s_o + row * a.dim + d, r), by, acc);
      }
    finish(row, d, m, l, acc);
  }
  __syncwarp();
  cluster_sync_all();                      // nobody leaves while its part is being read
}

int step_boxes(int dim, int rot) { return (dim + rot + 63) / 64; }
size_t step_fixed(int stages) { return 1024 + static_cast<size_t>(stages) * kTiedPage * 4 + 2 * kMaxStages * 8; }
// Two CTAs per SM where at least two pages of each fit.
int step_stages(int dim, int rot) {
  const size_t page = static_cast<size_t>(step_boxes(dim, rot)) * kTiedBox;
  for (size_t limit : {size_t(113) * 1024, size_t(227) * 1024}) {
    if (limit < 200 * 1024 && dim > 128) continue;
    int s = static_cast<int>((limit - step_fixed(kMaxStages)) / page);
    if (s > kMaxStages) s = kMaxStages;
    const size_t meet = (static_cast<size_t>(kWarps) * 16 * (dim + 2) + 32) * 4;
    if (s >= 2 && meet <= page * s) return s;
  }
  return 0;
}

template <int DB, int kSteps>
int launch_step(const StepParams& p, int segments, cudaStream_t st) {
  const cacheir_b200_tied_args& a = p.a;
  CUtensorMap map;
  if (!tied_encode(&map, a.pool, a.dim + a.rot_dims, static_cast<uint64_t>(a.num_slots) * a.kv_heads * kTiedPage)) return CACHEIR_B200_EUNSUPPORTED;
  const size_t smem = step_fixed(p.stages) + static_cast<size_t>(p.stages) * p.boxes * kTiedBox;
  auto kern = tied_step_kernel<DB, kSteps>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(p.splits, a.kv_heads * p.subs, segments);
  cfg.blockDim = dim3(kStepThreads, 1, 1);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = p.splits;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = p.splits > 1 ? 1 : 0;
  e = cudaLaunchKernelEx(&cfg, kern, map, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  return launch_status();
}

int head_groups(int group) { return (group + 15) / 16; }

}  // namespace

int tied_attention_status(bool reset) { return device_status_word(g_tied_status, reset); }

}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_tied_prepare(const cacheir_b200_tied_args* args, const void* q, long long q_stride, const void* k,
                                         long long k_stride, float eps, const float* rope_table, int rope_positions, void* q_out, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  if (args->rows <= 0) return 0;
  if (!tied_args_ok(*args) || !q || !k || !q_out || (args->rot_dims > 0 && !rope_table) || rope_positions <= 0) return CACHEIR_B200_EINVAL;
  const float2* table = reinterpret_cast<const float2*>(rope_table);
  const dim3 grid(args->rows, (args->heads + args->kv_heads + 7) / 8);
  if (grid.y > 65535) return CACHEIR_B200_ELIMIT;
  const bool vec = args->dim % 4 == 0 && args->rot_dims % 8 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && aligned_to(q, 16) &&
                   aligned_to(k, 8 * (args->dtype == CACHEIR_B200_F32 ? 2 : 1)) && aligned_to(args->pool, 16) && aligned_to(q_out, 16);
  CB200_HYBRID_DTYPE(args->dtype, {
    if (vec) tied_prepare_kernel<T, 4><<<grid, 256, 0, as_stream(stream)>>>(*args, static_cast<const T*>(q), q_stride, static_cast<const T*>(k),
                                                                           k_stride, eps, table, rope_positions, static_cast<T*>(q_out));
    else tied_prepare_kernel<T, 1><<<grid, 256, 0, as_stream(stream)>>>(*args, static_cast<const T*>(q), q_stride, static_cast<const T*>(k),
                                                                       k_stride, eps, table, rope_positions, static_cast<T*>(q_out));
  });
  return launch_status();
}

extern "C" int cacheir_b200_tied_attention_simple(const cacheir_b200_tied_args* args, const void* q, const void* gate, long long gate_stride,
                                                  void* out, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  if (args->rows <= 0) return 0;
  if (!tied_args_ok(*args) || !q || !out) return CACHEIR_B200_EINVAL;
  const size_t smem = static_cast<size_t>(2 * args->dim + args->rot_dims - tied_lead(args->rot_dims) + 128) * 4;
  if (smem > 48 * 1024) return CACHEIR_B200_ELIMIT;
  const dim3 grid(args->rows, args->heads);
  CB200_HYBRID_DTYPE(args->dtype, (tied_simple_kernel<T><<<grid, 128, smem, as_stream(stream)>>>(
                                      *args, static_cast<const T*>(q), static_cast<const T*>(gate), gate_stride, static_cast<T*>(out))));
  return launch_status();
}

extern "C" int cacheir_b200_tied_step_supported(int heads, int kv_heads, int dim, int rot_dims, int page_size, int dtype) {
  return dtype == CACHEIR_B200_BF16 && page_size == kTiedPage && kv_heads > 0 && heads % kv_heads == 0 && dim >= 8 && dim % 8 == 0 &&
         dim <= 256 && rot_dims >= 0 && rot_dims % 8 == 0 && rot_dims <= dim && step_stages(dim, rot_dims) > 0 &&
         static_cast<long long>(kv_heads) * head_groups(heads / kv_heads) <= 65535 ? 1 : 0;
}

extern "C" int cacheir_b200_tied_step_splits(int rows, int heads, int kv_heads, int window, int keep_first, int max_pages, int page_size) {
  if (rows <= 0 || heads <= 0 || kv_heads <= 0 || page_size <= 0) return 1;
  const long long units = static_cast<long long>(rows) * kv_heads * head_groups(heads / kv_heads);
  long long pages = (static_cast<long long>(window) + page_size - 2) / page_size + 1 + (keep_first + page_size - 1) / page_size;
  if (pages > max_pages) pages = max_pages;
  long long s = 2 * kNumSMs / units;
  if (s > pages / 2) s = pages / 2;      // at least two pages each
  return s < 1 ? 1 : static_cast<int>(s > kMaxSplits ? kMaxSplits : s);
}

extern "C" int cacheir_b200_tied_attention_step(const cacheir_b200_tied_args* args, const void* q, const void* gate, long long gate_stride,
                                                void* out, int splits, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_tied_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!tied_args_ok(a) || !q || !out || !a.decode || a.rows != a.segments) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_tied_step_supported(a.heads, a.kv_heads, a.dim, a.rot_dims, a.page_size, a.dtype)) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(q, 16) || !aligned_to(a.pool, 16) || !aligned_to(a.inv_rms, 16)) return CACHEIR_B200_EALIGN;
  if (splits <= 0) splits = cacheir_b200_tied_step_splits(a.rows, a.heads, a.kv_heads, a.window, a.keep_first, a.max_pages, a.page_size);
  if (splits > kMaxSplits || a.rows > 65535) return CACHEIR_B200_ELIMIT;
  StepParams p{};
  p.a = a;
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.gate_stride = gate_stride;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.score = tied_score(a.scale, a.cap);
  const int group = a.heads / a.kv_heads;
  p.subs = head_groups(group);
  p.heads_per_cta = (group + p.subs - 1) / p.subs;
  p.splits = splits;
  p.boxes = step_boxes(a.dim, a.rot_dims);
  p.stages = step_stages(a.dim, a.rot_dims);
  cudaStream_t st = as_stream(stream);
  const bool odd = (a.dim + a.rot_dims + 31) / 32 - a.rot_dims / 32 > (a.dim + 63) / 64 * 2;
  switch ((a.dim + 63) / 64) {
    case 1: return odd ? launch_step<1, 3>(p, a.rows, st) : launch_step<1, 2>(p, a.rows, st);
    case 2: return odd ? launch_step<2, 5>(p, a.rows, st) : launch_step<2, 4>(p, a.rows, st);
    case 3: return odd ? launch_step<3, 7>(p, a.rows, st) : launch_step<3, 6>(p, a.rows, st);
    default: return odd ? launch_step<4, 9>(p, a.rows, st) : launch_step<4, 8>(p, a.rows, st);
  }
}
