// Tied attention (a cached row is key and value) over a paged cache, sm_100a: preparation, the plain form, and decoding.
//
// prepare   one warp per head: root mean square, weights, rotation; queries go to a buffer, keys (and values) to their row.
// simple    any extents, float32 arithmetic: one CTA per (row, head).
// step      one CTA per (sequence, key/value head, split). Pages of 64 cached rows land in a ring as TMA boxes of 64 columns;
//           a row is read once and serves as key (columns from key_from on, times its reciprocal root mean square) and as
//           value (the first dim columns). Four warps take 16 rows of a page each with warp MMAs, the heads of the group
//           being the 16-row operand; they meet once per CTA, and splits meet in distributed shared memory.
#include "tied_attention.cuh"

namespace cb200 {
namespace {

__device__ int g_tied_status = 0;

struct PrepareParams {
  cacheir_b200_tied_args a;
  long long q_stride, k_stride, v_stride;
  const float* q_weight;        // per column of a head, or (whole) of the projection; NULL: ones
  const float* k_weight;
  const float2* table;
  int table_positions, rot_dims, head_dim;
  float eps;
};

// Entry c of a head: where it stands in a row, as rotated (c < rot_dims) or as projected.
__device__ __forceinline__ int key_column(const PrepareParams& p, bool tied, int c) {
  return tied ? (c < p.rot_dims ? p.a.dim + c : c) : p.a.dim + c;
}

// A warp per head. WHOLE: one block has all heads of a row and its root mean squares run over them; otherwise blocks share a row.
template <typename T, int VEC, bool WHOLE>
__global__ void __launch_bounds__(WHOLE ? 512 : 256)
tied_prepare_kernel(const PrepareParams p, const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, T* __restrict__ q_out) {
  constexpr int kWarpsHere = (WHOLE ? 512 : 256) / 32;
  __shared__ float s_part[2][kWarpsHere];
  const cacheir_b200_tied_args& a = p.a;
  const int row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int seg = a.row_seg[row], pos = a.positions[row], units = a.heads + a.kv_heads;      // query heads, then key heads
  if (seg < 0 || pos < 0 || pos >= p.table_positions || pos / a.page_size >= a.max_pages) return;
  const bool tied = v == nullptr;
  const int d = p.head_dim, half = p.rot_dims / 2, lead = tied_lead(a.key_from), group = a.heads / a.kv_heads;
  auto source = [&](int unit) {
    return unit < a.heads ? q + static_cast<size_t>(row) * p.q_stride + static_cast<size_t>(unit) * d
                          : k + static_cast<size_t>(row) * p.k_stride + static_cast<size_t>(unit - a.heads) * d;
  };
  auto squares = [&](const T* src) {
    float ss = 0.f;
    for (int c = lane * VEC; c < d; c += 32 * VEC) {
      float x[VEC];
      load_vec<T, VEC>(src + c, x);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(x[i], x[i], ss);
    }
    return ss;
  };
  float inv_q = 0.f, inv_k = 0.f;
  if (WHOLE) {
    float part[2] = {0.f, 0.f};
    for (int u = warp; u < units; u += kWarpsHere) part[u >= a.heads] += squares(source(u));
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      part[i] = warp_sum(part[i]);
      if (lane == 0) s_part[i][warp] = part[i];
    }
    __syncthreads();
    float total[2] = {0.f, 0.f};
    for (int w = 0; w < kWarpsHere; ++w) { total[0] += s_part[0][w]; total[1] += s_part[1][w]; }
    inv_q = 1.f / sqrtf(total[0] / static_cast<float>(a.heads * d) + p.eps);
    inv_k = 1.f / sqrtf(total[1] / static_cast<float>(a.kv_heads * d) + p.eps);
  }
  const int step = WHOLE ? kWarpsHere : units;
  for (int unit = (WHOLE ? 0 : blockIdx.y * kWarpsHere) + warp; unit < units; unit += step) {
    const bool key = unit >= a.heads;
    const int head = key ? unit - a.heads : unit, kv_head = key ? head : head / group;
    const T* src = source(unit);
    const float inv = WHOLE ? (key ? inv_k : inv_q) : 1.f / sqrtf(warp_sum(squares(src)) / static_cast<float>(d) + p.eps);
    // weights of this unit's own norm, and of the key that a query meets
    const float* own = key ? p.k_weight : p.q_weight;
    const float* met = p.k_weight;
    if (WHOLE && own) own += static_cast<size_t>(head) * d;
    if (WHOLE && met) met += static_cast<size_t>(kv_head) * d;
    T* dst;
    if (key) {
      const int slot = a.page_table[static_cast<size_t>(seg) * a.max_pages + pos / a.page_size];
      if (slot < 0 || slot >= a.num_slots) continue;
      const size_t at = (static_cast<size_t>(slot) * a.kv_heads + head) * a.page_size + pos % a.page_size;
      dst = static_cast<T*>(a.pool) + at * a.width;
      if (lane == 0) a.inv_rms[at] = inv;
      if (!tied) {
        const T* vs = v + static_cast<size_t>(row) * p.v_stride + static_cast<size_t>(head) * a.dim;
        for (int c = lane * VEC; c < a.dim; c += 32 * VEC) {
          float x[VEC];
          load_vec<T, VEC>(vs + c, x);
          store_vec<T, VEC>(dst + c, x);
        }
      }
    } else {
      dst = q_out + (static_cast<size_t>(row) * a.heads + head) * (a.width - lead) - lead;
      const float zero[VEC] = {};
      for (int c = lead + lane * VEC; c < a.key_from; c += 32 * VEC) store_vec<T, VEC>(dst + c, zero);
    }
    const float by = key ? 1.f : inv;        // keys keep their length: their factor lies beside the row
    const float2* cs = p.table + static_cast<size_t>(pos) * half;
    auto weigh = [&](const float* w, int c, float (&x)[VEC]) {
      if (!w) return;
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] *= w[c + i];
    };
    for (int c = lane * VEC; c < d; c += 32 * VEC) {
      float x[VEC];
      load_vec<T, VEC>(src + c, x);
      if (c < p.rot_dims) {
        if (key && tied) store_vec<T, VEC>(dst + c, x);          // the value
        const bool low = c < half;
        const int oc = low ? c + half : c - half;
        float other[VEC], r[VEC];
        load_vec<T, VEC>(src + oc, other);
        weigh(own, c, x);
        weigh(own, oc, other);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const float2 t = cs[(low ? c : oc) + i];
          r[i] = (low ? x[i] * t.x - other[i] * t.y : x[i] * t.x + other[i] * t.y) * by;
        }
        store_vec<T, VEC>(dst + key_column(p, tied, c), r);
      } else {
        if (!key) {                          // a key's unrotated entries stay as projected: their weights join the query's
          weigh(own, c, x);
          weigh(met, c, x);
#pragma unroll
          for (int i = 0; i < VEC; ++i) x[i] *= by;
        }
        store_vec<T, VEC>(dst + key_column(p, tied, c), x);
      }
    }
  }
}

// ---- plain form ------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
tied_simple_kernel(const cacheir_b200_tied_args a, const T* __restrict__ q, const T* __restrict__ gate, long long gate_stride,
                   T* __restrict__ out) {
  extern __shared__ float sm[];
  __shared__ float scratch[32];
  const int lead = tied_lead(a.key_from), width = a.width, qw = width - lead;
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
    const int width = a.width, lead = tied_lead(a.key_from), qw = width - lead;
    const int k_first = a.key_from / 32, last_piece = p.boxes * 2 - 1;      // (a piece behind the row meets zero queries: any data will do)
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

int step_boxes(int width) { return (width + 63) / 64; }
size_t step_fixed(int stages) { return 1024 + static_cast<size_t>(stages) * kTiedPage * 4 + 2 * kMaxStages * 8; }
// Two CTAs per SM where at least two pages of each fit.
int step_stages(int dim, int width) {
  const size_t page = static_cast<size_t>(step_boxes(width)) * kTiedBox;
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
  if (!tied_encode(&map, a.pool, a.width, static_cast<uint64_t>(a.num_slots) * a.kv_heads * kTiedPage)) return CACHEIR_B200_EUNSUPPORTED;
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

// 32-column pieces of a row that a query meets
constexpr int kMaxPieces = 9;
int step_pieces(int width, int key_from) { return (width + 31) / 32 - key_from / 32; }

int head_groups(int group) { return (group + 15) / 16; }

}  // namespace

int tied_attention_status(bool reset) { return device_status_word(g_tied_status, reset); }

}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_tied_prepare(const cacheir_b200_tied_args* args, const void* q, long long q_stride, const void* k,
                                         long long k_stride, const void* v, long long v_stride, int rot_dims, int whole,
                                         const float* q_weight, const float* k_weight, float eps, const float* rope_table,
                                         int rope_positions, void* q_out, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_tied_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!tied_args_ok(a) || !q || !k || !q_out || (rot_dims > 0 && !rope_table) || rope_positions <= 0) return CACHEIR_B200_EINVAL;
  const int d = v ? a.width - a.dim : a.dim;
  if (d <= 0 || rot_dims < 0 || rot_dims > d || rot_dims % 2 != 0 || a.key_from != (v ? a.dim : rot_dims) || (!v && a.width != a.dim + rot_dims))
    return CACHEIR_B200_EINVAL;
  const PrepareParams p{a, q_stride, k_stride, v_stride, q_weight, k_weight, reinterpret_cast<const float2*>(rope_table),
                        rope_positions, rot_dims, d, eps};
  const dim3 grid(a.rows, whole ? 1 : (a.heads + a.kv_heads + 7) / 8);
  if (grid.y > 65535) return CACHEIR_B200_ELIMIT;
  const int quad = 4 * (a.dtype == CACHEIR_B200_F32 ? 4 : 2);      // bytes of four elements
  const bool vec = d % 4 == 0 && a.dim % 4 == 0 && rot_dims % 8 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && aligned_to(q, quad) &&
                   aligned_to(k, quad) && (!v || (v_stride % 4 == 0 && aligned_to(v, quad))) && aligned_to(a.pool, quad) && aligned_to(q_out, quad);
#define CB200_PREPARE(VEC, WHOLE)                                                                                              \
  tied_prepare_kernel<T, VEC, WHOLE><<<grid, WHOLE ? 512 : 256, 0, as_stream(stream)>>>(                                        \
      p, static_cast<const T*>(q), static_cast<const T*>(k), static_cast<const T*>(v), static_cast<T*>(q_out))
  CB200_HYBRID_DTYPE(a.dtype, {
    if (vec && whole) CB200_PREPARE(4, true);
    else if (vec) CB200_PREPARE(4, false);
    else if (whole) CB200_PREPARE(1, true);
    else CB200_PREPARE(1, false);
  });
#undef CB200_PREPARE
  return launch_status();
}

extern "C" int cacheir_b200_tied_attention_simple(const cacheir_b200_tied_args* args, const void* q, const void* gate, long long gate_stride,
                                                  void* out, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  if (args->rows <= 0) return 0;
  if (!tied_args_ok(*args) || !q || !out) return CACHEIR_B200_EINVAL;
  const size_t smem = static_cast<size_t>(args->dim + args->width - tied_lead(args->key_from) + 128) * 4;
  if (smem > 48 * 1024) return CACHEIR_B200_ELIMIT;
  const dim3 grid(args->rows, args->heads);
  CB200_HYBRID_DTYPE(args->dtype, (tied_simple_kernel<T><<<grid, 128, smem, as_stream(stream)>>>(
                                      *args, static_cast<const T*>(q), static_cast<const T*>(gate), gate_stride, static_cast<T*>(out))));
  return launch_status();
}

extern "C" int cacheir_b200_tied_step_supported(int heads, int kv_heads, int dim, int width, int key_from, int page_size, int dtype) {
  return dtype == CACHEIR_B200_BF16 && page_size == kTiedPage && kv_heads > 0 && heads % kv_heads == 0 && dim >= 8 && dim % 8 == 0 &&
         dim <= 256 && width >= dim && width % 8 == 0 && key_from >= 0 && key_from % 8 == 0 && key_from < width &&
         step_pieces(width, key_from) <= kMaxPieces && step_stages(dim, width) > 0 &&
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
  if (!cacheir_b200_tied_step_supported(a.heads, a.kv_heads, a.dim, a.width, a.key_from, a.page_size, a.dtype)) return CACHEIR_B200_EUNSUPPORTED;
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
  p.boxes = step_boxes(a.width);
  p.stages = step_stages(a.dim, a.width);
  cudaStream_t st = as_stream(stream);
  const int pieces = step_pieces(a.width, a.key_from);
  switch ((a.dim + 63) / 64) {
    case 1: return pieces <= 2 ? launch_step<1, 2>(p, a.rows, st) : pieces == 3 ? launch_step<1, 3>(p, a.rows, st)
                 : pieces <= 5 ? launch_step<1, 5>(p, a.rows, st) : launch_step<1, kMaxPieces>(p, a.rows, st);
    case 2: return pieces <= 2 ? launch_step<2, 2>(p, a.rows, st) : pieces <= 4 ? launch_step<2, 4>(p, a.rows, st)
                 : pieces == 5 ? launch_step<2, 5>(p, a.rows, st) : launch_step<2, kMaxPieces>(p, a.rows, st);
    case 3: return pieces <= 3 ? launch_step<3, 3>(p, a.rows, st) : pieces <= 6 ? launch_step<3, 6>(p, a.rows, st)
                 : pieces == 7 ? launch_step<3, 7>(p, a.rows, st) : launch_step<3, kMaxPieces>(p, a.rows, st);
    default: return pieces <= 4 ? launch_step<4, 4>(p, a.rows, st) : pieces <= 8 ? launch_step<4, 8>(p, a.rows, st)
                 : launch_step<4, kMaxPieces>(p, a.rows, st);
  }
}
