// Tied attention over portions of prompts on the 5th-generation tensor cores, sm_100a.
//
// A CTA takes one or two tiles of 128 (token, head) rows of neighbouring tokens of one sequence; the heads of a tile share a
// key/value head. Pages of 64 cached rows land in a ring as TMA boxes of 64 columns and are used twice as they lie there:
//   S [rows, keys] = Q K^T     A = queries (M 128), B = the page's key columns (N 64), K-major
//   O [rows, dim] += P V       A = probabilities (M 128), B = the page's value columns read MN-major
// A softmax thread owns a row (a tensor-memory lane), so row sums need no exchange.
//   warp 0  copies      warp 1  MMA issue, tensor memory      warps 2..5, 6..9  softmax of tile 0, tile 1 (lane quarter = warp % 4)
//
// Where queries and keys have a known length (`reach`), |score| <= bound is known before any key is read. While exp(-2 bound) is
// far from underflow the softmax refers to the bound itself (FIXED): no running maximum, no rescaling. Otherwise a row's
// reference follows its maximum, and O is rescaled when that has grown by more than 2^8. The bound also makes the capped
// score a polynomial on a known interval: an odd one of five or eight terms, interpolated at Chebyshev nodes (TERMS).
#include "ragged.cuh"
#include "tied_attention.cuh"

namespace cb200 {
namespace {

__device__ int g_prompt_status = 0;

constexpr int kThreads = 320;
constexpr int kMaxStages = 6;
constexpr int kTile = 128;
constexpr int kTerms = 8;                   // of the polynomial, at most
constexpr float kStale = 8.f;

struct PromptParams {
  cacheir_b200_tied_args a;
  const __nv_bfloat16* gate;
  long long gate_stride;
  __nv_bfloat16* out;
  TiedScore score;
  float bound;                 // of |score| * log2 e
  float pre;                   // with a polynomial: raw product -> [-1, 1]
  float coef[kTerms];          // score * log2 e = y (coef[0] + coef[1] y^2 + ...)
  int subs, heads_per_cta, tokens_per_tile;
  int boxes, lead_boxes, stages;
  int n_cols;                  // output columns of the MMA
  int tmem_cols;
};

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
// MN-major operand as 128-byte swizzled rows: 64 columns a box, `box` bytes between boxes, 8-row groups 1024 bytes apart
__device__ __forceinline__ uint64_t smem_desc_mn_sw128(uint32_t addr, uint32_t box) {
  return static_cast<uint64_t>((addr >> 4) & 0x3FFF) | static_cast<uint64_t>((box >> 4) & 0x3FFF) << 16 |
         static_cast<uint64_t>(1024 >> 4) << 32 | static_cast<uint64_t>(1) << 46 | static_cast<uint64_t>(2) << 61;
}
__device__ __forceinline__ void tma_load_3d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int x, int y, int z) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(dst), "l"(reinterpret_cast<uint64_t>(map)), "r"(bar), "r"(x), "r"(y), "r"(z) : "memory");
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
// pairs of float32 in one instruction
using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pair(float lo, float hi) {
  f32x2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void unpair(f32x2 a, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(a)); }
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f32x2 add2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}

// Out of line: most waits find their barrier complete, and the loop's code would crowd theirs.
__device__ __noinline__ bool wait_long(uint32_t bar, uint32_t parity, int code) { return ptx::mbar_wait(bar, parity, &g_prompt_status, code); }

// TERMS: of the polynomial, 0: the formula
template <int TILES, bool FIXED, int TERMS>
__global__ void __launch_bounds__(kThreads, 1)
tied_prompt_kernel(const __grid_constant__ CUtensorMap tmap_kv, const __grid_constant__ CUtensorMap tmap_q, const PromptParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const cacheir_b200_tied_args& a = p.a;
  const int page_bytes = p.boxes * kTiedBox, q_boxes = p.boxes - p.lead_boxes, q_bytes = q_boxes * kTile * 128;
  uint8_t* s_kv = smem;                                         // [stages][boxes][64 rows][128 bytes], swizzled
  uint8_t* s_q = s_kv + p.stages * page_bytes;                  // [tiles][q_boxes][128 rows][128 bytes], swizzled
  uint8_t* s_p = s_q + TILES * q_bytes;                         // [page & 1][tiles][128 rows][128 bytes], swizzled
  float* s_inv = reinterpret_cast<float*>(s_p + 2 * TILES * kTile * 128);      // [stages][64]
  uint64_t* full = reinterpret_cast<uint64_t*>(s_inv + p.stages * kTiedPage);
  uint64_t* empty = full + kMaxStages;
  uint64_t* bar_q = empty + kMaxStages;
  // [page & 1][tile]: with one barrier per parity nobody can be two phases behind (a page's successor of the same parity
  // needs this page's probabilities from every thread)
  uint64_t* bar_s = bar_q + 1;             // scores in tensor memory
  uint64_t* bar_p = bar_s + 4;             // probabilities in shared memory
  uint64_t* bar_o = bar_p + 4;             // the page's output MMAs have retired
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar_o + 4);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = blockIdx.x / p.subs, sub = blockIdx.x % p.subs, group = a.heads / a.kv_heads;
  const int head0 = kvh * group + sub * p.heads_per_cta;
  const int nheads = min(p.heads_per_cta, group - sub * p.heads_per_cta);
  // the last tiles of a sequence have the most keys: they start first
  const RaggedItem item = find_item(a.cu_rows, a.segments, TILES * p.tokens_per_tile, gridDim.y - 1 - blockIdx.y);
  if (item.seg < 0) return;
  const int tiles = TILES == 2 && item.count > p.tokens_per_tile ? 2 : 1;
  const int pos0 = a.positions[item.row0];
  const TiedPages pages(a, pos0, pos0 + item.count - 1);
  const int n = pages.total;

  if (warp == 0 && lane == 0) {
    for (int s = 0; s < p.stages; ++s) { ptx::mbar_init(smem_addr(&full[s]), 1); ptx::mbar_init(smem_addr(&empty[s]), 1); }
    ptx::mbar_init(smem_addr(bar_q), 1);
    for (int t = 0; t < 4; ++t) {
      ptx::mbar_init(smem_addr(&bar_s[t]), 1);
      ptx::mbar_init(smem_addr(&bar_p[t]), 4);            // a warp each
      ptx::mbar_init(smem_addr(&bar_o[t]), 1);
    }
    ptx::mbar_fence_init();
  }
  if (warp == 1) ptx::tc_alloc(smem_addr(tmem_slot), p.tmem_cols);
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tmem = *tmem_slot;                             // output of tile t at column t * n_cols, scores behind
  const uint32_t tmem_s = tmem + TILES * p.n_cols;              // [page & 1][tile][64]
  bool ok = true;
  auto wait = [&](uint32_t bar, uint32_t parity, int code) {
    if (!ptx::mbar_try_wait(bar, parity)) ok = ok && wait_long(bar, parity, code);
  };

  if (warp == 0) {
    // ---------------- copies ----------------
    int slots = 0, issued = 0;
    if (lane == 0) {
      ptx::mbar_expect_tx(smem_addr(bar_q), tiles * q_boxes * p.heads_per_cta * p.tokens_per_tile * 128);
      for (int t = 0; t < tiles; ++t)
        for (int b = 0; b < q_boxes; ++b)
          tma_load_3d(smem_addr(s_q + t * q_bytes + b * kTile * 128), &tmap_q, smem_addr(bar_q), b * 64, head0, item.row0 + t * p.tokens_per_tile);
    }
    for (int it = 0; it < n; ++it) {
      if (it % 32 == 0) slots = it + lane < n ? tied_slot(a, item.seg, pages.page(it + lane)) : 0;
      const int slot = __shfl_sync(0xffffffffu, slots, it % 32);
      if (lane == 0) {
        const int s = it % p.stages;
        if (it >= p.stages) ok = ptx::mbar_wait(smem_addr(&empty[s]), ((it / p.stages) & 1) ^ 1, &g_prompt_status, (9 << 8) | 1);
        if (ok) {
          const uint32_t bar = smem_addr(&full[s]);
          const int unit = slot * a.kv_heads + kvh;
          ptx::mbar_expect_tx(bar, page_bytes + kTiedPage * 4);
          for (int b = 0; b < p.boxes; ++b)
            ptx::tma_load_2d(smem_addr(s_kv + s * page_bytes + b * kTiedBox), &tmap_kv, bar, b * 64, unit * kTiedPage);
          ptx::bulk_load(smem_addr(s_inv + s * kTiedPage), a.inv_rms + static_cast<size_t>(unit) * kTiedPage, kTiedPage * 4, bar);
          issued = it + 1;
        }
      }
      if (!__shfl_sync(0xffffffffu, ok ? 1 : 0, 0)) break;
    }
    if (lane == 0) {                     // nothing may still be on its way when the block ends, also after a wait that gave up
      ptx::mbar_wait(smem_addr(bar_q), 0, &g_prompt_status, (9 << 8) | 2);
      if (issued < n)
        for (int it = max(0, issued - p.stages); it < issued; ++it)
          ptx::mbar_wait(smem_addr(&full[it % p.stages]), (it / p.stages) & 1, &g_prompt_status, (9 << 8) | 3);
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------- MMA issue ----------------
    const uint32_t lead = lane == 0 ? 1u : 0u;
    const uint32_t id_s = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kTiedPage >> 3) << 17) | (static_cast<uint32_t>(kTile >> 4) << 24);
    const uint32_t id_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | (static_cast<uint32_t>(p.n_cols >> 3) << 17) |
                          (static_cast<uint32_t>(kTile >> 4) << 24);
    const uint64_t dq = ptx::smem_desc_sw128(smem_addr(s_q)), dk = ptx::smem_desc_sw128(smem_addr(s_kv + p.lead_boxes * kTiedBox));
    const uint64_t dp = ptx::smem_desc_sw128(smem_addr(s_p)), dv = smem_desc_mn_sw128(smem_addr(s_kv), kTiedBox);
    const uint32_t k_hi = static_cast<uint32_t>(dk >> 32), v_hi = static_cast<uint32_t>(dv >> 32);      // (dq, dk, dp share theirs)
    wait(smem_addr(bar_q), 0, (9 << 8) | 4);
    auto output = [&](int it) {
      const int s = it % p.stages;
      for (int t = 0; t < tiles; ++t) {
        wait(smem_addr(&bar_p[(it & 1) * 2 + t]), (it >> 1) & 1, (9 << 8) | 5);
        __syncwarp();
        ptx::tc_fence_after();
        const uint32_t pa = static_cast<uint32_t>(dp) + ((it & 1) * TILES + t) * (kTile * 128 >> 4), vb = static_cast<uint32_t>(dv) + s * (page_bytes >> 4);
#pragma unroll
        for (int j = 0; j < 4; ++j)          // 16 keys
          mma_f16_ss(lead, tmem + t * p.n_cols, pa + 2 * j, k_hi, vb + j * (2048 >> 4), v_hi, id_o, it > 0 || j > 0 ? 1u : 0u);
        if (lead) ptx::tc_commit(smem_addr(&bar_o[(it & 1) * 2 + t]));
        __syncwarp();
      }
      if (lead) ptx::tc_commit(smem_addr(&empty[s]));
      __syncwarp();
    };
#pragma unroll 1
    for (int it = 0; it < n; ++it) {       // (a score buffer is free: the probabilities of two pages before have been waited for)
      const int s = it % p.stages;
      wait(smem_addr(&full[s]), (it / p.stages) & 1, (9 << 8) | 6);
      __syncwarp();
      ptx::tc_fence_after();
#pragma unroll 1
      for (int t = 0; t < tiles; ++t) {
        const uint32_t d = tmem_s + ((it & 1) * TILES + t) * kTiedPage;
        uint32_t qa = static_cast<uint32_t>(dq) + t * (q_bytes >> 4), kb = static_cast<uint32_t>(dk) + s * (page_bytes >> 4);
#pragma unroll 1
        for (int b = 0; b < q_boxes; ++b) {
#pragma unroll
          for (int j = 0; j < 4; ++j)      // (columns beyond the row are zero in both operands)
            mma_f16_ss(lead, d, qa + 2 * j, k_hi, kb + 2 * j, k_hi, id_s, (b | j) > 0 ? 1u : 0u);
          qa += kTile * 128 >> 4;
          kb += kTiedBox >> 4;
        }
        if (lead) ptx::tc_commit(smem_addr(&bar_s[(it & 1) * 2 + t]));
        __syncwarp();
      }
      if (it > 0) output(it - 1);
    }
    output(n - 1);
  } else if (warp < 2 + 4 * tiles) {
    // ---------------- softmax: thread = row ----------------
    const int t = (warp - 2) >> 2, r = (warp & 3) * 32 + lane;
    const int tok = r / p.heads_per_cta, h = r % p.heads_per_cta;
    const int first = item.row0 + t * p.tokens_per_tile, count = min(p.tokens_per_tile, item.count - t * p.tokens_per_tile);
    const bool real = tok < count && h < nheads;
    const int tile_pos = pos0 + t * p.tokens_per_tile, rp = real ? tile_pos + tok : -1;
    const float sink = (a.sink && real) ? a.sink[head0 + h] * kLog2e : -1e30f;
    float m_ref = FIXED ? fmaxf(p.bound, sink) : sink;
    f32x2 l2 = pair(a.sink && real ? tied_ex2(sink - m_ref) : 0.f, 0.f);
    f32x2 coef[TERMS > 0 ? TERMS : 1];
#pragma unroll
    for (int k = 0; k < TERMS; ++k) coef[k] = pair(p.coef[k], p.coef[k]);
    const f32x2 pre = pair(p.pre, p.pre), minus_ref = pair(-m_ref, -m_ref);
    const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const int hi_row = rp, lo_row = rp - a.window;
    for (int it = 0; it < n; ++it) {
      const int s = it % p.stages, base = pages.page(it) * kTiedPage;
      const uint32_t scores = tmem_s + ((it & 1) * TILES + t) * kTiedPage + lanes;
      uint8_t* p_row = s_p + ((it & 1) * TILES + t) * kTile * 128 + r * 128;
      const float4* inv4 = reinterpret_cast<const float4*>(s_inv + s * kTiedPage);
      // (rows without a token may hold anything: a row of P reaches its own row of O only, which is not stored)
      const bool whole = base + kTiedPage - 1 <= tile_pos && (base > tile_pos + count - 1 - a.window || base + kTiedPage <= a.keep_first);
      if (it > 1) wait(smem_addr(&bar_o[(it & 1) * 2 + t]), ((it >> 1) & 1) ^ 1, (9 << 8) | 10);      // the P buffer is free
      wait(smem_addr(&full[s]), (it / p.stages) & 1, (9 << 8) | 8);
      wait(smem_addr(&bar_s[(it & 1) * 2 + t]), (it >> 1) & 1, (9 << 8) | 9);
      __syncwarp();
      ptx::tc_fence_after();
      // 16 scores * log2 e (FIXED: minus the reference) as pairs side by side, so that their chains overlap
      auto score16 = [&](int i0, f32x2 (&c)[8]) {
        float v[16];
        tmem_ld_x16(scores + i0, v);
        f32x2 u[8];
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
          const float4 f = inv4[i0 / 4 + j / 2];
          u[j] = mul2(pair(v[2 * j], v[2 * j + 1]), pair(f.x, f.y));
          u[j + 1] = mul2(pair(v[2 * j + 2], v[2 * j + 3]), pair(f.z, f.w));
        }
        if constexpr (TERMS > 0) {
          f32x2 w[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) u[j] = mul2(u[j], pre);
#pragma unroll
          for (int j = 0; j < 8; ++j) w[j] = mul2(u[j], u[j]);
#pragma unroll
          for (int j = 0; j < 8; ++j) c[j] = fma2(coef[TERMS - 1], w[j], coef[TERMS - 2]);
#pragma unroll
          for (int k = TERMS - 3; k >= 0; --k)
#pragma unroll
            for (int j = 0; j < 8; ++j) c[j] = fma2(c[j], w[j], coef[k]);
#pragma unroll
          for (int j = 0; j < 8; ++j) c[j] = FIXED ? fma2(c[j], u[j], minus_ref) : mul2(c[j], u[j]);
        } else {
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            float x, y;
            unpair(u[j], x, y);
            c[j] = pair(p.score(x), p.score(y));
            if (FIXED) c[j] = add2(c[j], minus_ref);
          }
        }
        if (!whole) {
          const int hi = hi_row - base - i0, lo = lo_row - base - i0, kept = a.keep_first - base - i0;
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            float x, y;
            unpair(c[j], x, y);
            if (!(2 * j <= hi && (2 * j > lo || 2 * j < kept))) x = -INFINITY;
            if (!(2 * j + 1 <= hi && (2 * j + 1 > lo || 2 * j + 1 < kept))) y = -INFINITY;
            c[j] = pair(x, y);
          }
        }
      };
      if constexpr (!FIXED) {
        float mx = -INFINITY, alpha = 1.f;
#pragma unroll 1
        for (int i0 = 0; i0 < kTiedPage; i0 += 16) {
          f32x2 c[8];
          score16(i0, c);
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            float x, y;
            unpair(c[j], x, y);
            mx = fmaxf(mx, fmaxf(x, y));
          }
        }
        if (mx > m_ref + (it == 0 ? 0.f : kStale)) {
          alpha = tied_ex2(m_ref - mx);
          m_ref = mx;
        }
        l2 = mul2(l2, pair(alpha, alpha));
        if (__any_sync(0xffffffffu, it > 0 && alpha != 1.f)) {        // rare: this warp's rows of O to the new references
          wait(smem_addr(&bar_o[((it - 1) & 1) * 2 + t]), ((it - 1) >> 1) & 1, (9 << 8) | 12);
          __syncwarp();
          ptx::tc_fence_after();
#pragma unroll 1
          for (int c = 0; c < p.n_cols; c += 16) {
            float o[16];
            tmem_ld_x16(tmem + t * p.n_cols + c + lanes, o);
#pragma unroll
            for (int j = 0; j < 16; ++j) o[j] *= alpha;
            tmem_st_x16(tmem + t * p.n_cols + c + lanes, o);
          }
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
      }
#pragma unroll
      for (int i0 = 0; i0 < kTiedPage; i0 += 16) {
        f32x2 c[8];
        score16(i0, c);
        uint32_t packed[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          float x, y;
          unpair(c[j], x, y);
          if (!FIXED) { x -= m_ref; y -= m_ref; }
          x = tied_ex2(x);
          y = tied_ex2(y);
          l2 = add2(l2, pair(x, y));
          packed[j] = pack_bf16(x, y);
        }
        *reinterpret_cast<uint4*>(p_row + (((i0 / 8) ^ (r & 7)) << 4)) = make_uint4(packed[0], packed[1], packed[2], packed[3]);
        *reinterpret_cast<uint4*>(p_row + (((i0 / 8 + 1) ^ (r & 7)) << 4)) = make_uint4(packed[4], packed[5], packed[6], packed[7]);
      }
      const int tail = pos0 + item.count - base;
      if (tail < kTiedPage && t == 0)        // rows behind the last token may hold anything: zero, so that 0 * row stays 0
        for (int i = threadIdx.x - 64; i < (kTiedPage - tail) * p.boxes * 8; i += kTile) {
          const int row = tail + i / (p.boxes * 8), c = i % (p.boxes * 8);
          *reinterpret_cast<uint4*>(s_kv + s * page_bytes + (c >> 3) * kTiedBox + row * 128 + (c & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");       // the tensor core reads what was just written
      ptx::tc_fence_before();
      __syncwarp();
      if (lane == 0) ptx::mbar_arrive(smem_addr(&bar_p[(it & 1) * 2 + t]));
    }
    const size_t row = first + tok, col0 = static_cast<size_t>(head0 + h) * a.dim;
    float l, l_odd;
    unpair(l2, l, l_odd);
    const float inv = 1.f / (l + l_odd);
    for (int c0 = 0; c0 < p.n_cols; c0 += 128) {
      uint4 g[16];                           // the gates travel while the last MMAs run
#pragma unroll
      for (int i = 0; i < 16; ++i)
        g[i] = p.gate && real && c0 + 8 * i < a.dim ? *reinterpret_cast<const uint4*>(p.gate + row * p.gate_stride + col0 + c0 + 8 * i) : make_uint4(0u, 0u, 0u, 0u);
      if (c0 == 0) wait(smem_addr(&bar_o[((n - 1) & 1) * 2 + t]), ((n - 1) >> 1) & 1, (9 << 8) | 11);
      __syncwarp();
      ptx::tc_fence_after();
#pragma unroll
      for (int c = 0; c < 128; c += 16) {
        if (c0 + c >= p.n_cols) break;
        float o[16];
        tmem_ld_x16(tmem + t * p.n_cols + c0 + c + lanes, o);
#pragma unroll
        for (int j = 0; j < 16; j += 8) {
          const uint32_t bits[4] = {g[(c + j) / 8].x, g[(c + j) / 8].y, g[(c + j) / 8].z, g[(c + j) / 8].w};
          float y[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const float gate = __uint_as_float(e & 1 ? bits[e / 2] & 0xffff0000u : bits[e / 2] << 16);
            y[e] = o[j + e] * inv * (p.gate ? sigmoid_exact(gate) : 1.f);
          }
          if (real && c0 + c + j < a.dim) VecIO<__nv_bfloat16, 8>::st(p.out + row * a.heads * a.dim + col0 + c0 + c + j, y);
        }
      }
    }
    __syncwarp();
  }
  ptx::tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    ptx::tc_fence_after();
    ptx::tc_dealloc(tmem, p.tmem_cols);
  }
}

constexpr size_t kSmemLimit = 227 * 1024;
int row_boxes(int width) { return (width + 63) / 64; }
size_t prompt_fixed(int tiles, int width, int key_from) {
  return 1024 + static_cast<size_t>(tiles) * (row_boxes(width) - key_from / 64 + 2) * kTile * 128 + kMaxStages * kTiedPage * 4 + (2 * kMaxStages + 13) * 8 + 16;
}
int prompt_stages(int tiles, int width, int key_from) {
  const size_t fixed = prompt_fixed(tiles, width, key_from), page = static_cast<size_t>(row_boxes(width)) * kTiedBox;
  const int s = fixed > kSmemLimit ? 0 : static_cast<int>((kSmemLimit - fixed) / page);
  return s > kMaxStages ? kMaxStages : (s >= 2 ? s : 0);
}

// Two tiles where tensor memory has room for their outputs and shared memory for their queries.
int prompt_tiles(int dim, int width, int key_from) { return dim <= 128 && prompt_stages(2, width, key_from) > 0 ? 2 : 1; }

// Odd polynomial for cap2 * tanh(reach * y) on [-1, 1]: y times the interpolant, at the Chebyshev nodes of [0, 1], of the
// even quotient as a function of y^2. Double precision. Returns the number of terms: the quotient's poles lie at
// y^2 = -(pi / 2 reach)^2, which puts the error near 2^-21 of cap2 or below; 0 where eight are not enough.
int fit_tanh(double cap2, double reach, float (&coef)[kTerms]) {
  if (!(reach > 0.0) || reach > 1.25) return 0;
  const int terms = reach <= 0.7 ? 5 : 8;
  const double pi = 3.14159265358979323846;
  double node[kTerms], table[kTerms];
  for (int i = 0; i < terms; ++i) {
    node[i] = 0.5 + 0.5 * cos((2 * i + 1) * pi / (2 * terms));
    const double y = sqrt(node[i]);
    table[i] = cap2 * tanh(reach * y) / y;
  }
  for (int k = 1; k < terms; ++k)                       // divided differences
    for (int i = terms - 1; i >= k; --i) table[i] = (table[i] - table[i - 1]) / (node[i] - node[i - k]);
  double c[kTerms] = {};
  for (int k = terms - 1; k >= 0; --k) {                // Newton form -> powers
    for (int i = terms - 1; i > 0; --i) c[i] = c[i - 1] - node[k] * c[i];
    c[0] = table[k] - node[k] * c[0];
  }
  for (int i = 0; i < terms; ++i) coef[i] = static_cast<float>(c[i]);
  return terms;
}

template <int TILES, bool FIXED, int TERMS>
int launch_prompt(const PromptParams& p, const void* q, int items, cudaStream_t st) {
  const cacheir_b200_tied_args& a = p.a;
  size_t smem = prompt_fixed(TILES, a.width, a.key_from) + static_cast<size_t>(p.stages) * p.boxes * kTiedBox;
  const size_t least = kSmemLimit / 2 + 1024;           // one CTA per SM: one that waited for tensor memory would be late
  if (smem < least) smem = least;
  CUtensorMap tkv, tq;
  if (!tied_encode(&tkv, a.pool, a.width, static_cast<uint64_t>(a.num_slots) * a.kv_heads * kTiedPage)) return CACHEIR_B200_EUNSUPPORTED;
  ptx::EncodeTiledFn fn = ptx::tensor_map_encoder();
  const cuuint64_t qw = a.width - tied_lead(a.key_from);
  const cuuint64_t dims[3] = {qw, static_cast<cuuint64_t>(a.heads), static_cast<cuuint64_t>(a.rows)};
  const cuuint64_t strides[2] = {qw * 2, qw * 2 * a.heads};
  const cuuint32_t box[3] = {64, static_cast<cuuint32_t>(p.heads_per_cta), static_cast<cuuint32_t>(p.tokens_per_tile)};
  const cuuint32_t elem_strides[3] = {1, 1, 1};
  if (fn(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(q), dims, strides, box, elem_strides, CU_TENSOR_MAP_INTERLEAVE_NONE,
         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return CACHEIR_B200_EUNSUPPORTED;
  auto kern = tied_prompt_kernel<TILES, FIXED, TERMS>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(a.kv_heads * p.subs, items), kThreads, smem, st>>>(tkv, tq, p);
  return launch_status();
}

template <int TILES>
int launch_tiles(const PromptParams& p, bool fixed, int terms, const void* q, int items, cudaStream_t st) {
  if (fixed && terms == 5) return launch_prompt<TILES, true, 5>(p, q, items, st);
  if (fixed && terms == 8) return launch_prompt<TILES, true, 8>(p, q, items, st);
  if (fixed) return launch_prompt<TILES, true, 0>(p, q, items, st);
  return launch_prompt<TILES, false, 0>(p, q, items, st);
}

}  // namespace

int tied_prompt_status(bool reset) { return device_status_word(g_prompt_status, reset); }

}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_tied_prompt_supported(int heads, int kv_heads, int dim, int width, int key_from, int page_size, int dtype) {
  return dtype == CACHEIR_B200_BF16 && page_size == kTiedPage && kv_heads > 0 && heads % kv_heads == 0 && dim >= 8 && dim % 8 == 0 &&
         dim <= 256 && width >= dim && width % 8 == 0 && key_from >= 0 && key_from % 8 == 0 && key_from < width &&
         prompt_stages(1, width, key_from) > 0 ? 1 : 0;
}

extern "C" int cacheir_b200_tied_attention_prompt(const cacheir_b200_tied_args* args, const void* q, const void* gate, long long gate_stride,
                                                  void* out, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_tied_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!tied_args_ok(a) || !q || !out || !a.cu_rows) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_tied_prompt_supported(a.heads, a.kv_heads, a.dim, a.width, a.key_from, a.page_size, a.dtype)) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(q, 16) || !aligned_to(a.pool, 16) || !aligned_to(a.inv_rms, 16) || !aligned_to(out, 16) ||
      (gate && (!aligned_to(gate, 16) || gate_stride % 8 != 0)))
    return CACHEIR_B200_EALIGN;
  PromptParams p{};
  p.a = a;
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.gate_stride = gate_stride;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.score = tied_score(a.scale, a.cap);
  // a little room for the operands' rounding
  const double most = a.reach * 1.02, reach = most * fabs(static_cast<double>(a.scale));
  const double bound = a.cap > 0.f ? a.cap * tanh(reach / a.cap) : reach;
  p.bound = static_cast<float>(bound * kLog2e);
  const bool fixed = a.reach > 0.f && 2.0 * bound * kLog2e <= 100.0;
  int terms = 0;
  if (a.cap > 0.f && fixed) {
    p.pre = static_cast<float>((a.scale < 0.f ? -1.0 : 1.0) / most);
    terms = fit_tanh(static_cast<double>(a.cap) * kLog2e, reach / a.cap, p.coef);
  }
  const int group = a.heads / a.kv_heads, tiles = prompt_tiles(a.dim, a.width, a.key_from);
  p.subs = (group + kTile - 1) / kTile;
  p.heads_per_cta = (group + p.subs - 1) / p.subs;
  p.tokens_per_tile = kTile / p.heads_per_cta;
  p.boxes = row_boxes(a.width);
  p.lead_boxes = a.key_from / 64;
  p.stages = prompt_stages(tiles, a.width, a.key_from);
  p.n_cols = (a.dim + 15) / 16 * 16;
  const int cols = tiles * (p.n_cols + 2 * kTiedPage);
  p.tmem_cols = cols <= 128 ? 128 : cols <= 256 ? 256 : 512;
  const int items = ragged_items(a.rows, a.segments, tiles * p.tokens_per_tile);
  if (items > 65535) return CACHEIR_B200_ELIMIT;
  return tiles == 2 ? launch_tiles<2>(p, fixed, terms, q, items, as_stream(stream)) : launch_tiles<1>(p, fixed, terms, q, items, as_stream(stream));
}
