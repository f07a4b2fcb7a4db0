// Talking-heads attention over portions of prompts on the 5th-generation tensor cores, sm_100a.
//
// A CTA takes one or two tiles of 128 (token, head) rows of neighbouring tokens of one sequence; the heads of a tile share a
// key/value head. With mixed queries (talking_prepare) a row's mixed scores are one product with whole cached key rows, so for a
// block of 128 keys
//   S [rows, 128] = Q K^T      a GEMM over all key columns: boxes of 64 columns of the queries and of the keys pass through a ring
//   O [rows, vdim] += P V      A = probabilities in tensor memory, where the scores were; B = the block's values read MN-major
// A softmax thread owns a row (a tensor-memory lane). Its reference starts at the score 0 that has no value and follows the row's
// maximum when that has grown by more than 2^8.
//   warp 0  copies      warp 1  MMA issue, tensor memory      warps 2..5, 6..9  softmax of tile 0, tile 1 (lane quarter = warp % 4)
// The next block's scores are issued when this block's output products have retired: the score product is the long part (all
// key/value heads' columns), and its operands travel during the softmax.
#include "ragged.cuh"
#include "talking_attention.cuh"

namespace cb200 {
namespace {

__device__ int g_prompt_status = 0;

constexpr int kThreads = 320;
constexpr int kMaxStages = 6;
constexpr int kTile = 128;                  // rows
constexpr int kKeys = 128;                  // of a block: two pages
constexpr int kQBox = kTile * 128, kKBox = kTalkPage * 128;
constexpr float kStale = 8.f;

struct PromptParams {
  cacheir_b200_talking_args a;
  __nv_bfloat16* out;
  int subs, heads_per_cta, tokens_per_tile;
  int steps;                   // boxes of a key row
  int v_boxes, stages;
  int n_cols;                  // output columns of the MMA
  int tmem_cols;
};

// All lanes come here; one issues.
__device__ __forceinline__ void mma_ss(uint32_t lead, uint32_t tmem_d, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(tmem_d), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate), "r"(lead) : "memory");
}
__device__ __forceinline__ void mma_ts(uint32_t lead, uint32_t tmem_d, uint32_t tmem_a, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(tmem_d), "r"(tmem_a), "l"(b_desc), "r"(idesc), "r"(accumulate), "r"(lead) : "memory");
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
__device__ __forceinline__ void tmem_ld_x32(uint32_t taddr, float (&v)[32]) {
  uint32_t r[32];
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,"
      "%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
        "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]),
        "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]),
        "=r"(r[30]), "=r"(r[31])
      : "r"(taddr) : "memory");
#pragma unroll
  for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(r[i]);      // (nobody reads them before a tc_wait_ld)
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
__device__ __forceinline__ void tmem_st_x16(uint32_t taddr, const uint32_t (&v)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]),
      "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]) : "memory");
}
__device__ __forceinline__ void tmem_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// pairs of float32 in one instruction
using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pair(float lo, float hi) {
  f32x2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void unpair(f32x2 a, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(a)); }
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

template <int TILES>
__global__ void __launch_bounds__(kThreads, 1)
talking_prompt_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                      const __grid_constant__ CUtensorMap tmap_v, const PromptParams p) {
  constexpr int kStage = TILES * kQBox + 2 * kKBox;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const cacheir_b200_talking_args& a = p.a;
  uint8_t* s_v = smem + p.stages * kStage;                      // [2 pages][v_boxes][64 rows][128 bytes], swizzled
  const int v_page = p.v_boxes * kKBox;
  uint64_t* full = reinterpret_cast<uint64_t*>(s_v + 2 * v_page);
  uint64_t* empty = full + kMaxStages;
  uint64_t* full_v = empty + kMaxStages;
  uint64_t* bar_s = full_v + 1;            // scores in tensor memory
  uint64_t* bar_p = bar_s + 1;             // [tile] probabilities in tensor memory
  uint64_t* bar_o = bar_p + 2;             // the block's output MMAs have retired
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar_o + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = blockIdx.x / p.subs, sub = blockIdx.x % p.subs, group = a.heads / a.kv_heads;
  const int head0 = kvh * group + sub * p.heads_per_cta;
  const int nheads = min(p.heads_per_cta, group - sub * p.heads_per_cta);
  // the last tiles of a sequence have the most keys: they start first
  const RaggedItem item = find_item(a.cu_rows, a.segments, TILES * p.tokens_per_tile, gridDim.y - 1 - blockIdx.y);
  if (item.seg < 0) return;
  const int tiles = TILES == 2 && item.count > p.tokens_per_tile ? 2 : 1;
  const int pos0 = a.positions[item.row0], pos_last = pos0 + item.count - 1;
  const int page_lo = max(0, pos0 - a.window + 1) / kTalkPage, n = (pos_last / kTalkPage - page_lo + 2) / 2;      // blocks

  if (warp == 0 && lane == 0) {
    for (int s = 0; s < p.stages; ++s) { ptx::mbar_init(smem_addr(&full[s]), 1); ptx::mbar_init(smem_addr(&empty[s]), 1); }
    ptx::mbar_init(smem_addr(full_v), 1);
    ptx::mbar_init(smem_addr(bar_s), 1);
    for (int t = 0; t < 2; ++t) ptx::mbar_init(smem_addr(&bar_p[t]), 4);      // a warp each
    ptx::mbar_init(smem_addr(bar_o), 1);
    ptx::mbar_fence_init();
  }
  if (warp == 1) ptx::tc_alloc(smem_addr(tmem_slot), p.tmem_cols);
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tmem = *tmem_slot;                             // output of tile t at column t * n_cols, scores behind
  const uint32_t tmem_s = tmem + TILES * p.n_cols;              // [tile][128]
  bool ok = true;
  auto wait = [&](uint32_t bar, uint32_t parity, int code) {
    if (!ptx::mbar_try_wait(bar, parity)) ok = ok && wait_long(bar, parity, code);
  };

  if (warp == 0) {
    // ---------------- copies ----------------
    if (lane == 0) {
      const uint32_t q_bytes = p.heads_per_cta * p.tokens_per_tile * 128;
      int issued = 0, values = 0;
      for (int it = 0; it < n && ok; ++it) {
        int row[2];
        for (int i = 0; i < 2; ++i) row[i] = talk_slot(a, item.seg, page_lo + 2 * it + i) * kTalkPage;
        for (int k = 0; k < p.steps; ++k) {
          const int s = issued % p.stages;
          if (issued >= p.stages) ok = ptx::mbar_wait(smem_addr(&empty[s]), ((issued / p.stages) & 1) ^ 1, &g_prompt_status, (11 << 8) | 1);
          if (!ok) break;
          const uint32_t bar = smem_addr(&full[s]), dst = smem_addr(smem + s * kStage);
          ptx::mbar_expect_tx(bar, tiles * q_bytes + 2 * kKBox);
          for (int t = 0; t < tiles; ++t)
            tma_load_3d(dst + t * kQBox, &tmap_q, bar, k * 64, head0, item.row0 + t * p.tokens_per_tile);
          for (int i = 0; i < 2; ++i) ptx::tma_load_2d(dst + TILES * kQBox + i * kKBox, &tmap_k, bar, k * 64, row[i]);
          ++issued;
        }
        if (ok && it > 0) ok = ptx::mbar_wait(smem_addr(bar_o), (it - 1) & 1, &g_prompt_status, (11 << 8) | 2);      // the values are spent
        if (!ok) break;
        ptx::mbar_expect_tx(smem_addr(full_v), 2 * v_page);
        for (int i = 0; i < 2; ++i)
          for (int b = 0; b < p.v_boxes; ++b)
            ptx::tma_load_2d(smem_addr(s_v + i * v_page + b * kKBox), &tmap_v, smem_addr(full_v), kvh * a.vdim + b * 64, row[i]);
        values = it + 1;
      }
      // nothing may still be on its way when the block ends, also after a wait that gave up
      if (!ok) {
        for (int i = max(0, issued - p.stages); i < issued; ++i)
          ptx::mbar_wait(smem_addr(&full[i % p.stages]), (i / p.stages) & 1, &g_prompt_status, (11 << 8) | 3);
        if (values > 0) ptx::mbar_wait(smem_addr(full_v), (values - 1) & 1, &g_prompt_status, (11 << 8) | 4);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------- MMA issue ----------------
    const uint32_t lead = lane == 0 ? 1u : 0u;
    const uint32_t id_s = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kKeys >> 3) << 17) | (static_cast<uint32_t>(kTile >> 4) << 24);
    const uint32_t id_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | (static_cast<uint32_t>(p.n_cols >> 3) << 17) |
                          (static_cast<uint32_t>(kTile >> 4) << 24);
    int used = 0;
    for (int it = 0; it < n; ++it) {
      if (it > 0) wait(smem_addr(bar_o), (it - 1) & 1, (11 << 8) | 5);      // scores take the place of probabilities that have been read
#pragma unroll 1
      for (int k = 0; k < p.steps; ++k, ++used) {
        const int s = used % p.stages;
        wait(smem_addr(&full[s]), (used / p.stages) & 1, (11 << 8) | 6);
        __syncwarp();
        ptx::tc_fence_after();
        const uint32_t at = smem_addr(smem + s * kStage);
        for (int t = 0; t < tiles; ++t)
#pragma unroll
          for (int j = 0; j < 4; ++j)          // (columns beyond the row are zero in both operands)
            mma_ss(lead, tmem_s + t * kKeys, ptx::smem_desc_sw128(at + t * kQBox + j * 32), ptx::smem_desc_sw128(at + TILES * kQBox + j * 32), id_s,
                   (k | j) > 0 ? 1u : 0u);
        if (lead) ptx::tc_commit(smem_addr(&empty[s]));
        __syncwarp();
      }
      if (lead) ptx::tc_commit(smem_addr(bar_s));
      __syncwarp();
      wait(smem_addr(full_v), it & 1, (11 << 8) | 7);
      for (int t = 0; t < tiles; ++t) {
        wait(smem_addr(&bar_p[t]), it & 1, (11 << 8) | 8);
        __syncwarp();
        ptx::tc_fence_after();
#pragma unroll
        for (int j = 0; j < kKeys / 16; ++j)
          mma_ts(lead, tmem + t * p.n_cols, tmem_s + t * kKeys + j * 8, smem_desc_mn_sw128(smem_addr(s_v) + (j / 4) * v_page + (j % 4) * 2048, kKBox), id_o,
                 it > 0 || j > 0 ? 1u : 0u);
      }
      if (lead) ptx::tc_commit(smem_addr(bar_o));
      __syncwarp();
    }
  } else if (warp < 2 + 4 * tiles) {
    // ---------------- softmax: thread = row ----------------
    const int t = (warp - 2) >> 2, r = (warp & 3) * 32 + lane;
    const int tok = r / p.heads_per_cta, h = r % p.heads_per_cta;
    const int first = item.row0 + t * p.tokens_per_tile, count = min(p.tokens_per_tile, item.count - t * p.tokens_per_tile);
    const bool real = tok < count && h < nheads;
    const int tile_pos = pos0 + t * p.tokens_per_tile, rp = real ? tile_pos + tok : -1;
    const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t scores = tmem_s + t * kKeys + lanes, outputs = tmem + t * p.n_cols + lanes;
    const float scale = fabsf(a.scale) * kTalkLog2e;      // (its sign is the queries')
    float m_ref = 0.f, l = 1.f;                    // the score 0 that has no value
    for (int it = 0; it < n; ++it) {
      const int base = (page_lo + 2 * it) * kTalkPage;
      // (rows without a token may hold anything: a row of P reaches its own row of O only, which is not stored)
      const bool whole = base + kKeys - 1 <= tile_pos && base > tile_pos + count - 1 - a.window;
      const int hi = rp - base, lo = rp - a.window - base;      // seen: lo < key <= hi
      auto mask = [&](int c, float (&v)[2][32]) {
#pragma unroll
        for (int j = 0; j < 64; ++j)
          if (!(c + j <= hi && c + j > lo)) v[j >> 5][j & 31] = -INFINITY;
      };
      wait(smem_addr(bar_s), it & 1, (11 << 8) | 9);
      __syncwarp();
      ptx::tc_fence_after();
      float mx = -INFINITY;
#pragma unroll 1
      for (int c = 0; c < kKeys; c += 64) {
        float v[2][32], m[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
        tmem_ld_x32(scores + c, v[0]);
        tmem_ld_x32(scores + c + 32, v[1]);
        ptx::tc_wait_ld();
        if (!whole) mask(c, v);
#pragma unroll
        for (int j = 0; j < 64; ++j) m[j & 3] = fmaxf(m[j & 3], v[j >> 5][j & 31]);
        mx = fmaxf(mx, fmaxf(fmaxf(m[0], m[1]), fmaxf(m[2], m[3])));
      }
      mx *= scale;
      float alpha = 1.f;
      if (mx > m_ref + kStale) {
        alpha = talk_ex2(m_ref - mx);
        m_ref = mx;
        l *= alpha;
      }
      if (__any_sync(0xffffffffu, it > 0 && alpha != 1.f)) {      // rare: this warp's rows of O to the new references
#pragma unroll 1
        for (int c = 0; c < p.n_cols; c += 16) {
          float o[16];
          uint32_t bits[16];
          tmem_ld_x16(outputs + c, o);
#pragma unroll
          for (int j = 0; j < 16; ++j) bits[j] = __float_as_uint(o[j] * alpha);
          tmem_st_x16(outputs + c, bits);
        }
      }
      const f32x2 factor = pair(scale, scale), minus_ref = pair(-m_ref, -m_ref);
      f32x2 sum[2] = {pair(0.f, 0.f), pair(0.f, 0.f)};
#pragma unroll 1
      for (int c = 0; c < kKeys; c += 64) {
        float v[2][32];
        tmem_ld_x32(scores + c, v[0]);
        tmem_ld_x32(scores + c + 32, v[1]);
        ptx::tc_wait_ld();
        if (!whole) mask(c, v);
        uint32_t packed[2][16];
#pragma unroll
        for (int j = 0; j < 64; j += 2) {
          float x, y;
          unpair(fma2(pair(v[j >> 5][j & 31], v[j >> 5][(j & 31) + 1]), factor, minus_ref), x, y);
          x = talk_ex2(x);
          y = talk_ex2(y);
          sum[(j >> 1) & 1] = add2(sum[(j >> 1) & 1], pair(x, y));
          packed[j >> 5][(j & 31) / 2] = pack_bf16(x, y);
        }
        tmem_st_x16(scores + c / 2, packed[0]);       // (behind what this thread has read)
        tmem_st_x16(scores + c / 2 + 16, packed[1]);
      }
      float part[4];
      unpair(sum[0], part[0], part[1]);
      unpair(sum[1], part[2], part[3]);
      l += (part[0] + part[1]) + (part[2] + part[3]);
      tmem_wait_st();
      const int tail = pos_last + 1 - base;
      if (tail < kKeys && t == 0) {                // values behind the last token may be anything: zero, so that 0 * value stays 0
        wait(smem_addr(full_v), it & 1, (11 << 8) | 10);
        for (int i = threadIdx.x - 64; i < (kKeys - tail) * p.v_boxes * 8; i += kTile) {
          const int row = tail + i / (p.v_boxes * 8), c = i % (p.v_boxes * 8);
          *reinterpret_cast<uint4*>(s_v + (row >> 6) * v_page + (c >> 3) * kKBox + (row & 63) * 128 + (c & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");       // the tensor core reads what was just written
      }
      ptx::tc_fence_before();
      __syncwarp();
      if (lane == 0) ptx::mbar_arrive(smem_addr(&bar_p[t]));
    }
    const size_t row = first + tok, col0 = static_cast<size_t>(head0 + h) * a.vdim;
    const float inv = 1.f / l;
    wait(smem_addr(bar_o), (n - 1) & 1, (11 << 8) | 11);
    __syncwarp();
    ptx::tc_fence_after();
    for (int c = 0; c < p.n_cols; c += 16) {
      float o[16];
      tmem_ld_x16(outputs + c, o);
#pragma unroll
      for (int j = 0; j < 16; j += 8) {
        float y[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] = o[j + e] * inv;
        if (real && c + j < a.vdim) VecIO<__nv_bfloat16, 8>::st(p.out + row * a.heads * a.vdim + col0 + c + j, y);
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
int prompt_tiles(int vdim) { return vdim <= 128 ? 2 : 1; }      // tensor memory: outputs and 128 scores each
size_t prompt_fixed(int vdim) { return 1024 + static_cast<size_t>(2) * ((vdim + 63) / 64) * kKBox + (2 * kMaxStages + 5) * 8 + 16; }
int prompt_stages(int vdim) {
  const int s = static_cast<int>((kSmemLimit - prompt_fixed(vdim)) / (prompt_tiles(vdim) * kQBox + 2 * kKBox));
  return s > kMaxStages ? kMaxStages : s;
}

template <int TILES>
int launch_prompt(const PromptParams& p, const void* q, int items, cudaStream_t st) {
  const cacheir_b200_talking_args& a = p.a;
  const size_t smem = prompt_fixed(a.vdim) + static_cast<size_t>(p.stages) * (TILES * kQBox + 2 * kKBox);
  CUtensorMap tq, tk, tv;
  const cuuint64_t width = static_cast<cuuint64_t>(a.kv_heads) * a.dim, cached = static_cast<cuuint64_t>(a.num_slots) * kTalkPage;
  if (!talk_encode(&tk, a.keys, width, cached, kTalkPage) || !talk_encode(&tv, a.values, static_cast<uint64_t>(a.kv_heads) * a.vdim, cached, kTalkPage))
    return CACHEIR_B200_EUNSUPPORTED;
  ptx::EncodeTiledFn fn = ptx::tensor_map_encoder();
  const cuuint64_t dims[3] = {width, static_cast<cuuint64_t>(a.heads), static_cast<cuuint64_t>(a.rows)};
  const cuuint64_t strides[2] = {width * 2, width * 2 * a.heads};
  const cuuint32_t box[3] = {64, static_cast<cuuint32_t>(p.heads_per_cta), static_cast<cuuint32_t>(p.tokens_per_tile)};
  const cuuint32_t elem_strides[3] = {1, 1, 1};
  if (fn(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(q), dims, strides, box, elem_strides, CU_TENSOR_MAP_INTERLEAVE_NONE,
         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return CACHEIR_B200_EUNSUPPORTED;
  auto kern = talking_prompt_kernel<TILES>;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(a.kv_heads * p.subs, items), kThreads, smem, st>>>(tq, tk, tv, p);
  return launch_status();
}

}  // namespace

int talking_prompt_status(bool reset) { return device_status_word(g_prompt_status, reset); }

}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_talking_prompt_supported(int heads, int kv_heads, int dim, int vdim, int page_size, int dtype) {
  return dtype == CACHEIR_B200_BF16 && page_size == kTalkPage && kv_heads > 0 && heads % kv_heads == 0 && dim >= 8 && dim % 8 == 0 && vdim >= 8 &&
         vdim % 8 == 0 && vdim <= 256 && (static_cast<long long>(heads) * dim + static_cast<long long>(heads) * heads) * 4 <= 200 * 1024 ? 1 : 0;
}

extern "C" int cacheir_b200_talking_prompt(const cacheir_b200_talking_args* args, const void* mixed_q, void* out, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_talking_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!talk_args_ok(a) || !mixed_q || !out || !a.cu_rows) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_talking_prompt_supported(a.heads, a.kv_heads, a.dim, a.vdim, a.page_size, a.dtype)) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(mixed_q, 16) || !aligned_to(a.keys, 16) || !aligned_to(a.values, 16) || !aligned_to(out, 16)) return CACHEIR_B200_EALIGN;
  PromptParams p{};
  p.a = a;
  p.out = static_cast<__nv_bfloat16*>(out);
  const int group = a.heads / a.kv_heads, tiles = prompt_tiles(a.vdim);
  p.subs = (group + kTile - 1) / kTile;
  p.heads_per_cta = (group + p.subs - 1) / p.subs;
  p.tokens_per_tile = kTile / p.heads_per_cta;
  p.steps = (a.kv_heads * a.dim + 63) / 64;
  p.v_boxes = (a.vdim + 63) / 64;
  p.stages = prompt_stages(a.vdim);
  p.n_cols = (a.vdim + 15) / 16 * 16;
  const int cols = tiles * (p.n_cols + kKeys);
  p.tmem_cols = cols <= 256 ? 256 : 512;
  const int items = ragged_items(a.rows, a.segments, tiles * p.tokens_per_tile);
  if (items > 65535) return CACHEIR_B200_ELIMIT;
  return tiles == 2 ? launch_prompt<2>(p, mixed_q, items, as_stream(stream)) : launch_prompt<1>(p, mixed_q, items, as_stream(stream));
}
