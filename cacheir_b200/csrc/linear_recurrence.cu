// Linear recurrence S <- decay S + take k v^T, o = S^T q per head, float32 state carried per sequence slot, sm_100a.
// decay is a constant per head and take one; or (GATED) both belong to the token and the head, given as logarithms, and where
// somebody normalises o a vector n <- decay n + take k runs along, of which q . n is kept. Neighbouring heads may share q and k,
// and a multiple of v may be added to o.
//
// simple   any extents and types: one CTA per (sequence, head, 32 value columns) walks the tokens, state in shared memory
// step     decode: one CTA per (sequence, head) streams the state once (16-byte accesses), HBM bound
// chunked  prompts, bf16 operands on the tensor cores, 64 tokens at a time. With D_ij = decay^(i-j) for j <= i:
//            O = diag(decay^(i+1)) Q S + ((Q K^T) o D) V        S' = decay^n S + K^T diag(decay^(n-1-j)) V
//          The state stays in float32 registers; whatever is float32 by nature and has to enter an MMA (the state, the
//          decayed scores, the decayed values) goes in as a sum of two bf16 numbers. With many heads a CTA runs through its whole
//          sequence, the next chunk's inputs travelling ahead; with few, sequences are cut into pieces of
//          64 to 256 tokens that run in parallel: a first pass finds every piece's own contribution, a scan turns these into the
//          pieces' initial states, and the main pass starts from them. GATED: with c the running sum of log decays in a
//          chunk, decay^(i-j) becomes exp(c_i - c_j + log take_j), and so on; n rides with the first value columns.
// gates    matrix memory: log decay and log take from gate logits, relative to a running maximum (a scan over the tokens)
// memory   matrix memory, decode: gates, state, normaliser, the head's norm and the output gate in one pass over the state
// space    state space: its gates for prompts, and one decoded token (gates and recurrence in one pass over the state)
#include "cacheir_b200_recurrence.h"
#include "hybrid_common.cuh"
#include "ragged.cuh"

namespace cb200 {
namespace {

constexpr int kPowers = 65;
constexpr int kChunk = 64;
constexpr int kPiece = 256;        // tokens of a piece at most, and of a step that is not cut
constexpr int kWide = 8, kNarrow = 4;      // 8-column tiles of the values per CTA of the chunked form: in pieces, whole sequences

using Args = cacheir_b200_recurrence_args;

// A slot: [heads][dim][vdim] state; with gates also [heads][dim] normaliser and [heads] running maxima behind it.
__device__ __forceinline__ float* slot_base(const Args& a, int seg) {
  const int slot = min(max(a.slots[seg], 0), a.num_slots - 1);
  return a.state + static_cast<size_t>(slot) * a.slot_stride;
}
__device__ __forceinline__ float* slot_state(const Args& a, int seg, int h) {
  return slot_base(a, seg) + static_cast<size_t>(h) * a.dim * a.vdim;
}
__device__ __forceinline__ float* slot_normaliser(const Args& a, int seg, int h) {
  return slot_base(a, seg) + static_cast<size_t>(a.heads) * a.dim * a.vdim + static_cast<size_t>(h) * a.dim;
}
__device__ __forceinline__ float* slot_maximum(const Args& a, int seg, int h) {
  return slot_base(a, seg) + static_cast<size_t>(a.heads) * a.dim * (a.vdim + 1) + h;
}

__device__ __forceinline__ int key_head(const Args& a, int h) { return a.key_heads > 0 ? h / (a.heads / a.key_heads) : h; }

template <typename T, bool GATED>
__global__ void __launch_bounds__(256)
recurrence_simple_kernel(const Args a) {
  extern __shared__ float sm[];
  float* s_state = sm;                       // [dim][32]
  float* s_k = s_state + a.dim * 32;         // [dim]
  float* s_q = s_k + a.dim;                  // [dim]
  float* s_n = s_q + a.dim;                  // [dim]
  float* s_red = s_n + a.dim;                // [8][32]
  const int seg = blockIdx.x, h = blockIdx.y;
  const int row0 = a.cu_rows[seg], row1 = a.cu_rows[seg + 1];
  if (row0 >= row1) return;
  const int lane = threadIdx.x & 31, group = threadIdx.x >> 5;
  const int col = blockIdx.z * 32 + lane;
  const bool col_ok = col < a.vdim;
  float* state = slot_state(a, seg, h);
  const bool fresh = a.positions[row0] == 0;
  for (int d = group; d < a.dim; d += 8)
    s_state[d * 32 + lane] = (fresh || !col_ok) ? 0.f : state[static_cast<size_t>(d) * a.vdim + col];
  const bool first = GATED && a.normaliser && blockIdx.z == 0;        // this block also has the normaliser
  const int kh = key_head(a, h);
  const float skip = a.skip ? a.skip[h] : 0.f;
  if (first)
    for (int d = threadIdx.x; d < a.dim; d += 256) s_n[d] = fresh ? 0.f : slot_normaliser(a, seg, h)[d];
  float decay = GATED ? 0.f : a.decay_pow[h * kPowers + 1], take = 1.f;
  for (int row = row0; row < row1; ++row) {
    __syncthreads();
    if (GATED) {
      decay = expf(a.log_decay[static_cast<size_t>(row) * a.heads + h]);
      take = expf(a.log_take[static_cast<size_t>(row) * a.heads + h]);
    }
    const size_t off = static_cast<size_t>(row) * a.stride;
    for (int d = threadIdx.x; d < a.dim; d += 256) {
      s_k[d] = Elem<T>::ld(static_cast<const T*>(a.k) + off + static_cast<size_t>(kh) * a.dim + d) * take;
      s_q[d] = Elem<T>::ld(static_cast<const T*>(a.q) + off + static_cast<size_t>(kh) * a.dim + d) * (GATED ? a.q_scale : 1.f);
    }
    const float v = col_ok ? Elem<T>::ld(static_cast<const T*>(a.v) + off + static_cast<size_t>(h) * a.vdim + col) : 0.f;
    __syncthreads();
    float o = 0.f;
    for (int d = group; d < a.dim; d += 8) {
      const float s = fmaf(s_state[d * 32 + lane], decay, s_k[d] * v);
      s_state[d * 32 + lane] = s;
      o = fmaf(s, s_q[d], o);
    }
    s_red[group * 32 + lane] = o;
    __syncthreads();
    if (group == 0 && col_ok) {
      float t = skip * v;
#pragma unroll
      for (int g = 0; g < 8; ++g) t += s_red[g * 32 + lane];
      Elem<T>::st(static_cast<T*>(a.out) + (static_cast<size_t>(row) * a.heads + h) * a.vdim + col, t);
    }
    if (first) {
      float nq = 0.f;
      for (int d = threadIdx.x; d < a.dim; d += 256) {
        const float n = fmaf(s_n[d], decay, s_k[d]);
        s_n[d] = n;
        nq = fmaf(n, s_q[d], nq);
      }
      nq = block_sum_all(nq, s_red + 256);
      if (threadIdx.x == 0) a.normaliser[static_cast<size_t>(row) * a.heads + h] = nq;
    }
  }
  if (first)
    for (int d = threadIdx.x; d < a.dim; d += 256) slot_normaliser(a, seg, h)[d] = s_n[d];
  if (col_ok)
    for (int d = group; d < a.dim; d += 8) state[static_cast<size_t>(d) * a.vdim + col] = s_state[d * 32 + lane];
}

template <typename T>
__global__ void __launch_bounds__(256)
recurrence_step_kernel(const Args a) {
  __shared__ float4 s_red[256];
  extern __shared__ float s_kq[];           // [2][dim]
  const int seg = blockIdx.x, h = blockIdx.y;
  const int row = a.cu_rows[seg];
  const int groups_per_row = a.vdim / 4;                 // float4 columns
  const int lanes_rows = 256 / groups_per_row;           // state rows per pass
  const int cg = threadIdx.x % groups_per_row, rg = threadIdx.x / groups_per_row;
  const bool active = rg < lanes_rows;
  const size_t off = static_cast<size_t>(row) * a.stride;
  for (int d = threadIdx.x; d < a.dim; d += 256) {
    s_kq[d] = Elem<T>::ld(static_cast<const T*>(a.k) + off + static_cast<size_t>(h) * a.dim + d);
    s_kq[a.dim + d] = Elem<T>::ld(static_cast<const T*>(a.q) + off + static_cast<size_t>(h) * a.dim + d);
  }
  float v[4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
    v[i] = active ? Elem<T>::ld(static_cast<const T*>(a.v) + off + static_cast<size_t>(h) * a.vdim + cg * 4 + i) : 0.f;
  const bool fresh = a.positions[row] == 0;
  const float decay = fresh ? 0.f : a.decay_pow[h * kPowers + 1];
  float4* state = reinterpret_cast<float4*>(slot_state(a, seg, h));
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  constexpr int U = 8;                                   // loads in flight per thread
  for (int d0 = rg; active && d0 < a.dim; d0 += U * lanes_rows) {
    float4 s[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int d = d0 + u * lanes_rows;
      s[u] = (d < a.dim && !fresh) ? state[static_cast<size_t>(d) * groups_per_row + cg] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int d = d0 + u * lanes_rows;
      if (d >= a.dim) break;
      const float k = s_kq[d], q = s_kq[a.dim + d];
      s[u].x = fmaf(s[u].x, decay, k * v[0]); s[u].y = fmaf(s[u].y, decay, k * v[1]);
      s[u].z = fmaf(s[u].z, decay, k * v[2]); s[u].w = fmaf(s[u].w, decay, k * v[3]);
      state[static_cast<size_t>(d) * groups_per_row + cg] = s[u];
      o.x = fmaf(s[u].x, q, o.x); o.y = fmaf(s[u].y, q, o.y); o.z = fmaf(s[u].z, q, o.z); o.w = fmaf(s[u].w, q, o.w);
    }
  }
  s_red[threadIdx.x] = o;
  __syncthreads();
  if (rg == 0) {
    for (int g = 1; g < lanes_rows; ++g) {
      const float4 t = s_red[g * groups_per_row + cg];
      o.x += t.x; o.y += t.y; o.z += t.z; o.w += t.w;
    }
    T* dst = static_cast<T*>(a.out) + (static_cast<size_t>(row) * a.heads + h) * a.vdim + cg * 4;
    Elem<T>::st(dst, o.x); Elem<T>::st(dst + 1, o.y); Elem<T>::st(dst + 2, o.z); Elem<T>::st(dst + 3, o.w);
  }
}

// ---- chunked form ----------------------------------------------------------------------------------------------------
// Between the passes: every piece's state [pieces][heads][dim][vdim]; with gates also its normaliser [pieces][heads][dim] and
// the sum of its log decays [pieces][heads].
struct PieceSpace {
  float* state;
  float* normaliser;
  float* log_decay;
};
PieceSpace piece_space(const Args& a, float* ws, int items) {
  float* n = ws + static_cast<size_t>(items) * a.heads * a.dim * a.vdim;
  return {ws, n, n + static_cast<size_t>(items) * a.heads * a.dim};
}

// MT = 16-row state tiles per warp (dim <= 64 MT), NC = 8-column tiles. AHEAD: two buffers of inputs, the next chunk's travel while
// this one's products run.
template <int MT, int NC, bool LOCAL, bool GATED, bool AHEAD>
__global__ void __launch_bounds__(128)
recurrence_chunk_kernel(const Args a, const PieceSpace ws, int piece_rows) {
  constexpr int kCols = NC * 8, kPitchV = kCols + 8;      // (rows 16 bytes over a multiple of 32: conflict-free)
  constexpr int kBuffers = AHEAD ? 2 : 1;
  extern __shared__ __align__(16) uint8_t raw[];
  const int dim = a.dim;
  const int pitch = dim + 8;
  __nv_bfloat16* q_bufs = reinterpret_cast<__nv_bfloat16*>(raw);     // [buffers][64][pitch]
  __nv_bfloat16* k_bufs = q_bufs + kBuffers * kChunk * pitch;        // [buffers][64][pitch]
  __nv_bfloat16* v_bufs = k_bufs + kBuffers * kChunk * pitch;        // [buffers][64][kPitchV]
  __nv_bfloat16* s_dv = v_bufs + kBuffers * kChunk * kPitchV;        // [2][64][kPitchV] decayed values, hi | lo
  __nv_bfloat16* s_s = s_dv + 2 * kChunk * kPitchV;                  // [2][dim][kPitchV] state, hi | lo
  __shared__ float s_pow[kPowers];
  __shared__ float s_cum[kChunk], s_take[kChunk], s_left[kChunk];      // log decays summed, log take, weight in the chunk's last state
  __shared__ float s_n[2][128];                       // the normaliser before and after a chunk
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, v0 = blockIdx.z * kCols;

  const RaggedItem it = find_item(a.cu_rows, a.segments, piece_rows, blockIdx.x);
  if (it.seg < 0) return;
  const bool alone = it.last && static_cast<int>(blockIdx.x) == it.first;     // the segment is a single piece
  if (LOCAL && it.last) return;                                               // nobody needs its contribution
  if (!GATED)
    for (int i = threadIdx.x; i < kPowers; i += 128) s_pow[i] = a.decay_pow[h * kPowers + i];

  float st[MT][NC][4];         // state rows (warp + 4 t)*16 .. +15, columns v0 .. v0 + kCols - 1
  float* state = slot_state(a, it.seg, h);
  float* piece = ws.state + (static_cast<size_t>(blockIdx.x) * a.heads + h) * dim * a.vdim;
  float* piece_n = ws.normaliser + (static_cast<size_t>(blockIdx.x) * a.heads + h) * dim;
  const float* init = alone ? state : piece;
  const bool zero = LOCAL || (alone && a.positions[it.row0] == 0);
  const int cols = min(kCols, a.vdim - v0);
  const bool first = GATED && a.normaliser && blockIdx.z == 0;        // this block also has the normaliser
  const int kh = key_head(a, h);
  const float skip = a.skip ? a.skip[h] : 0.f;
  float sum = 0.f;                                    // of the piece's log decays
  if (first && static_cast<int>(threadIdx.x) < dim)
    s_n[0][threadIdx.x] = zero ? 0.f : (alone ? slot_normaliser(a, it.seg, h) : piece_n)[threadIdx.x];
#pragma unroll
  for (int t = 0; t < MT; ++t)
#pragma unroll
    for (int n = 0; n < NC; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = (warp + 4 * t) * 16 + (lane >> 2) + e * 8, c = n * 8 + (lane & 3) * 2;
        float2 x = make_float2(0.f, 0.f);
        if (!zero && d < dim && c < cols) x = *reinterpret_cast<const float2*>(init + static_cast<size_t>(d) * a.vdim + v0 + c);
        st[t][n][e * 2] = x.x;
        st[t][n][e * 2 + 1] = x.y;
      }
  __syncthreads();

  const int kc = dim / 8;      // 16-byte pieces per q / k row
  const int r_first = static_cast<int>(threadIdx.x) / kc, c_first = static_cast<int>(threadIdx.x) % kc, r_step = 128 / kc, c_step = 128 % kc;
  auto next_piece = [&](int& r, int& c) {      // 128 pieces further
    r += r_step;
    c += c_step;
    if (c >= kc) { c -= kc; ++r; }
  };
  int now = 0;                 // which of s_n is the current one
  float ahead[4] = {};         // warp 0: the next chunk's log decays and log takes, two rows per lane
  auto fetch_gates = [&](int r0) {
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int r = r0 + u * 32 + lane;
      const size_t at = (static_cast<size_t>(it.row0) + r) * a.heads + h;
      ahead[u] = r < it.count ? a.log_decay[at] : 0.f;
      ahead[2 + u] = r < it.count ? a.log_take[at] : 0.f;
    }
  };
  if (GATED && warp == 0) fetch_gates(0);
  // AHEAD: a chunk's inputs, asynchronously; a thread copies the values that it decays
  auto fetch = [&](int r0) {
    const int buf = (r0 / kChunk) & 1, n = min(kChunk, it.count - r0);
    const size_t base = static_cast<size_t>(it.row0 + r0);
    auto copy = [&](__nv_bfloat16* dst, const void* src, size_t off, bool there) {      // (what lies behind the end is zero)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(static_cast<const __nv_bfloat16*>(src) + off),
                   "r"(there ? 16 : 0) : "memory");
    };
    for (int r = r_first, c = c_first; r < kChunk; next_piece(r, c)) {
      const size_t off = (base + min(r, n - 1)) * a.stride + static_cast<size_t>(kh) * dim + c * 8;
      copy(q_bufs + (buf * kChunk + r) * pitch + c * 8, a.q, off, r < n);
      copy(k_bufs + (buf * kChunk + r) * pitch + c * 8, a.k, off, r < n);
    }
    for (int i = threadIdx.x; i < kChunk * NC; i += 128) {
      const int r = i / NC, c = i % NC;
      const bool there = r < n && c * 8 < cols;
      copy(v_bufs + (buf * kChunk + r) * kPitchV + c * 8, a.v, (base + min(r, n - 1)) * a.stride + static_cast<size_t>(h) * a.vdim + v0 + (there ? c * 8 : 0), there);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (AHEAD) fetch(0);
  for (int r0 = 0; r0 < it.count; r0 += kChunk) {
    const int n = min(kChunk, it.count - r0);
    const size_t base = static_cast<size_t>(it.row0 + r0);
    const int buf = AHEAD ? (r0 / kChunk) & 1 : 0;
    __nv_bfloat16* s_q = q_bufs + buf * kChunk * pitch;
    __nv_bfloat16* s_k = k_bufs + buf * kChunk * pitch;
    __nv_bfloat16* s_v = v_bufs + buf * kChunk * kPitchV;
    if (GATED) {
      if (warp == 0) {
        float c[2], take[2], last = 0.f;
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          c[u] = ahead[u];
          take[u] = ahead[2 + u];
#pragma unroll
          for (int off = 1; off < 32; off <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, c[u], off);
            if (lane >= off) c[u] += up;
          }
          c[u] += last;
          last = __shfl_sync(0xffffffffu, c[u], 31);
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int r = u * 32 + lane;
          s_cum[r] = c[u];
          s_take[r] = take[u];
          s_left[r] = r < n ? __expf(last - c[u] + take[u]) : 0.f;
        }
        if (r0 + kChunk < it.count) fetch_gates(r0 + kChunk);
      }
      __syncthreads();
    }
    if (AHEAD) asm volatile("cp.async.wait_group 0;" ::: "memory");
    for (int r = AHEAD ? kChunk : r_first, c = c_first; r < kChunk; next_piece(r, c)) {
      uint4 q = make_uint4(0u, 0u, 0u, 0u), k = q;
      if (r < n) {
        const size_t off = (base + r) * a.stride + static_cast<size_t>(kh) * dim + c * 8;
        if (!LOCAL) q = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.q) + off);
        k = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.k) + off);
      }
      if (!LOCAL) *reinterpret_cast<uint4*>(s_q + r * pitch + c * 8) = q;
      *reinterpret_cast<uint4*>(s_k + r * pitch + c * 8) = k;
    }
    for (int i = threadIdx.x; i < kChunk * NC; i += 128) {
      const int r = i / NC, c = i % NC;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (AHEAD) v = *reinterpret_cast<const uint4*>(s_v + r * kPitchV + c * 8);
      else if (r < n && c * 8 < cols)
        v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.v) + (base + r) * a.stride + static_cast<size_t>(h) * a.vdim + v0 + c * 8);
      if (!LOCAL && !AHEAD) *reinterpret_cast<uint4*>(s_v + r * kPitchV + c * 8) = v;
      const float f = GATED ? s_left[r] : s_pow[max(n - 1 - r, 0)];
      const uint32_t* w = reinterpret_cast<const uint32_t*>(&v);
      uint4 hi, lo;
      uint32_t* hw = reinterpret_cast<uint32_t*>(&hi);
      uint32_t* lw = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float h0, l0, h1, l1;
        split_bf16(__uint_as_float(w[j] << 16) * f, &h0, &l0);
        split_bf16(__uint_as_float(w[j] & 0xffff0000u) * f, &h1, &l1);
        hw[j] = pack_bf16(h0, h1);
        lw[j] = pack_bf16(l0, l1);
      }
      *reinterpret_cast<uint4*>(s_dv + r * kPitchV + c * 8) = hi;
      *reinterpret_cast<uint4*>(s_dv + (kChunk + r) * kPitchV + c * 8) = lo;
    }
    if (!LOCAL) {
#pragma unroll
      for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int nn = 0; nn < NC; ++nn)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int d = (warp + 4 * t) * 16 + (lane >> 2) + e * 8, c = nn * 8 + (lane & 3) * 2;
            if (d < dim) {
              float h0, l0, h1, l1;
              split_bf16(st[t][nn][e * 2], &h0, &l0);
              split_bf16(st[t][nn][e * 2 + 1], &h1, &l1);
              *reinterpret_cast<uint32_t*>(s_s + d * kPitchV + c) = pack_bf16(h0, h1);
              *reinterpret_cast<uint32_t*>(s_s + (dim + d) * kPitchV + c) = pack_bf16(l0, l1);
            }
          }
    }
    __syncthreads();
    if (AHEAD && r0 + kChunk < it.count) fetch(r0 + kChunk);

    if (!LOCAL && warp * 16 < n) {
      float o[NC][4];
#pragma unroll
      for (int nn = 0; nn < NC; ++nn)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[nn][e] = 0.f;
      float sc[8][4];
#pragma unroll
      for (int nn = 0; nn < 8; ++nn)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nn][e] = 0.f;
      const uint32_t qa = smem_addr(s_q) + ((warp * 16 + (lane & 15)) * pitch + (lane >> 4) * 8) * 2;
      const uint32_t ka = smem_addr(s_k) + (((lane & 7) + ((lane >> 4) << 3)) * pitch + ((lane >> 3) & 1) * 8) * 2;
      const uint32_t sa = smem_addr(s_s) + (((lane & 7) + ((lane >> 3) & 1) * 8) * kPitchV + (lane >> 4) * 8) * 2;
      for (int k = 0; k < dim / 16; ++k) {
        uint32_t af[4];
        ldsm_x4(qa + k * 32, af);
#pragma unroll
        for (int nn = 0; nn < 8; nn += 2) {
          if (nn <= 2 * warp + 1) {                   // keys up to this band's last row
            uint32_t bf[4];
            ldsm_x4(ka + nn * 8 * pitch * 2 + k * 32, bf);
            mma_bf16(sc[nn], af, bf[0], bf[1]);
            mma_bf16(sc[nn + 1], af, bf[2], bf[3]);
          }
        }
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int nn = 0; nn < NC; nn += 2) {
            uint32_t bf[4];
            ldsm_x4_t(sa + ((part * dim + k * 16) * kPitchV + nn * 8) * 2, bf);
            mma_bf16(o[nn], af, bf[0], bf[1]);
            mma_bf16(o[nn + 1], af, bf[2], bf[3]);
          }
      }
      const int i0 = warp * 16 + (lane >> 2);
      const float f0 = GATED ? __expf(s_cum[i0]) * a.q_scale : s_pow[i0 + 1], f1 = GATED ? __expf(s_cum[i0 + 8]) * a.q_scale : s_pow[i0 + 9];
      float nq[2] = {0.f, 0.f};
      if (first) {                                    // q . (n before the chunk): a quarter of the entries per lane of the row
        for (int d = lane & 3; d < dim; d += 4) {
          nq[0] = fmaf(__bfloat162float(s_q[i0 * pitch + d]), s_n[now][d], nq[0]);
          nq[1] = fmaf(__bfloat162float(s_q[(i0 + 8) * pitch + d]), s_n[now][d], nq[1]);
        }
        nq[0] *= f0;
        nq[1] *= f1;
      }
#pragma unroll
      for (int nn = 0; nn < NC; ++nn) {
        o[nn][0] *= f0; o[nn][1] *= f0; o[nn][2] *= f1; o[nn][3] *= f1;
      }
      const uint32_t va = smem_addr(s_v) + (((lane & 7) + ((lane >> 3) & 1) * 8) * kPitchV + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {                // 16 keys
        if (kk > warp) continue;
        float d[2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = i0 + (e >> 1) * 8, j = kk * 16 + u * 8 + (lane & 3) * 2 + (e & 1);
            if (GATED) d[u][e] = j <= i ? sc[2 * kk + u][e] * (__expf(s_cum[i] - s_cum[j] + s_take[j]) * a.q_scale) : 0.f;
            else d[u][e] = j <= i ? sc[2 * kk + u][e] * s_pow[i - j] : 0.f;
            if (GATED) nq[e >> 1] += d[u][e];
          }
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float h0, l0, h1, l1;
            split_bf16(d[u][e * 2], &h0, &l0);
            split_bf16(d[u][e * 2 + 1], &h1, &l1);
            hi[u * 2 + e] = pack_bf16(h0, h1);
            lo[u * 2 + e] = pack_bf16(l0, l1);
          }
#pragma unroll
        for (int nn = 0; nn < NC; nn += 2) {
          uint32_t bf[4];
          ldsm_x4_t(va + (kk * 16 * kPitchV + nn * 8) * 2, bf);
          mma_bf16(o[nn], hi, bf[0], bf[1]);
          mma_bf16(o[nn + 1], hi, bf[2], bf[3]);
          mma_bf16(o[nn], lo, bf[0], bf[1]);
          mma_bf16(o[nn + 1], lo, bf[2], bf[3]);
        }
      }
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = i0 + e * 8;
        if (first) {
          nq[e] += __shfl_xor_sync(0xffffffffu, nq[e], 1);
          nq[e] += __shfl_xor_sync(0xffffffffu, nq[e], 2);
          if ((lane & 3) == 0 && i < n) a.normaliser[(base + i) * a.heads + h] = nq[e];
        }
        if (i < n && a.skip) {
#pragma unroll
          for (int nn = 0; nn < NC; ++nn) {
            const uint32_t v2 = *reinterpret_cast<const uint32_t*>(s_v + i * kPitchV + nn * 8 + (lane & 3) * 2);
            o[nn][e * 2] = fmaf(skip, __uint_as_float(v2 << 16), o[nn][e * 2]);
            o[nn][e * 2 + 1] = fmaf(skip, __uint_as_float(v2 & 0xffff0000u), o[nn][e * 2 + 1]);
          }
        }
        if (i < n) {
          __nv_bfloat16* dst = out + ((base + i) * a.heads + h) * a.vdim + v0;
#pragma unroll
          for (int nn = 0; nn < NC; ++nn) {
            const int c = nn * 8 + (lane & 3) * 2;
            if (c < cols) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(o[nn][e * 2], o[nn][e * 2 + 1]);
          }
        }
      }
    }

    // S' = decay^n S + K^T (decayed V)
    const float fn = GATED ? __expf(s_cum[n - 1]) : s_pow[n];
    if (GATED) sum += s_cum[n - 1];
    const uint32_t kt = smem_addr(s_k) + (((lane & 7) + ((lane >> 4) & 1) * 8) * pitch + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t dv = smem_addr(s_dv) + (((lane & 7) + ((lane >> 3) & 1) * 8) * kPitchV + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      const int m0 = (warp + 4 * t) * 16;
      if (m0 >= dim) continue;
#pragma unroll
      for (int nn = 0; nn < NC; ++nn)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[t][nn][e] *= fn;
#pragma unroll
      for (int k = 0; k < kChunk / 16; ++k) {
        uint32_t af[4];
        ldsm_x4_t(kt + (k * 16 * pitch + m0) * 2, af);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int nn = 0; nn < NC; nn += 2) {
            uint32_t bf[4];
            ldsm_x4_t(dv + ((part * kChunk + k * 16) * kPitchV + nn * 8) * 2, bf);
            mma_bf16(st[t][nn], af, bf[0], bf[1]);
            mma_bf16(st[t][nn + 1], af, bf[2], bf[3]);
          }
      }
    }
    if (first) {
      const int d = threadIdx.x;
      if (d < dim) {                                  // (rows behind the last are zero)
        float x[4] = {s_n[now][d] * fn, 0.f, 0.f, 0.f};
#pragma unroll 4
        for (int r = 0; r < kChunk; r += 4)
#pragma unroll
          for (int u = 0; u < 4; ++u) x[u] = fmaf(s_left[r + u], __bfloat162float(s_k[(r + u) * pitch + d]), x[u]);
        s_n[now ^ 1][d] = (x[0] + x[1]) + (x[2] + x[3]);
      }
    }
    now ^= 1;
    __syncthreads();
  }

  float* dst = LOCAL ? piece : state;
  if (LOCAL || it.last) {
    if (first && static_cast<int>(threadIdx.x) < dim) (LOCAL ? piece_n : slot_normaliser(a, it.seg, h))[threadIdx.x] = s_n[now][threadIdx.x];
    if (LOCAL && GATED && blockIdx.z == 0 && threadIdx.x == 0) ws.log_decay[static_cast<size_t>(blockIdx.x) * a.heads + h] = sum;
#pragma unroll
    for (int t = 0; t < MT; ++t)
#pragma unroll
      for (int n = 0; n < NC; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int d = (warp + 4 * t) * 16 + (lane >> 2) + e * 8, c = n * 8 + (lane & 3) * 2;
          if (d < dim && c < cols)
            *reinterpret_cast<float2*>(dst + static_cast<size_t>(d) * a.vdim + v0 + c) = make_float2(st[t][n][e * 2], st[t][n][e * 2 + 1]);
        }
  }
}

// Contributions of a segment's pieces -> their initial states (in place). A thread has four neighbouring entries; several
// pieces' are requested before the first is used.
template <bool GATED>
__global__ void __launch_bounds__(256)
recurrence_scan_kernel(const Args a, const PieceSpace ws, int piece_rows) {
  constexpr int kAhead = 8;
  __shared__ float s_f[256];
  const int seg = blockIdx.x, h = blockIdx.y;
  int first = 0;
  for (int s = 0; s < seg; ++s) first += (a.cu_rows[s + 1] - a.cu_rows[s] + piece_rows - 1) / piece_rows;
  const int rows = a.cu_rows[seg + 1] - a.cu_rows[seg];
  const int pieces = (rows + piece_rows - 1) / piece_rows;
  if (pieces < 2) return;
  const size_t plane = static_cast<size_t>(a.dim) * a.vdim;
  float constant = 1.f;
  if (!GATED)
    for (int i = 0; i < piece_rows; i += 64) constant *= a.decay_pow[h * kPowers + 64];
  const bool fresh = a.positions[a.cu_rows[seg]] == 0;
  const size_t e = (static_cast<size_t>(blockIdx.z) * 256 + threadIdx.x) * 4;
  const bool mine = e < plane;
  float4* w = reinterpret_cast<float4*>(ws.state + (static_cast<size_t>(first) * a.heads + h) * plane + (mine ? e : 0));
  const size_t stride = a.heads * plane / 4;
  float4 run = make_float4(0.f, 0.f, 0.f, 0.f);
  if (mine && !fresh) run = *reinterpret_cast<const float4*>(slot_state(a, seg, h) + e);
  const bool norm = GATED && a.normaliser && blockIdx.z == 0 && static_cast<int>(threadIdx.x) < a.dim;      // (dim <= 128)
  float* wn = ws.normaliser + (static_cast<size_t>(first) * a.heads + h) * a.dim + threadIdx.x;
  float run_n = norm && !fresh ? slot_normaliser(a, seg, h)[threadIdx.x] : 0.f;
  for (int base = 0; base < pieces; base += 256) {
    if (GATED) {
      __syncthreads();
      const int i = base + threadIdx.x;
      if (i < pieces - 1) s_f[threadIdx.x] = expf(ws.log_decay[static_cast<size_t>(first + i) * a.heads + h]);
      __syncthreads();
    }
    const int stop = min(pieces, base + 256);
    for (int i0 = base; i0 < stop; i0 += kAhead) {
      float4 own[kAhead];
      float own_n[kAhead];
#pragma unroll
      for (int u = 0; u < kAhead; ++u) {                 // (nobody needs the last piece's contribution: it has none)
        const bool there = i0 + u < min(stop, pieces - 1);
        own[u] = there && mine ? w[(i0 + u) * stride] : make_float4(0.f, 0.f, 0.f, 0.f);
        own_n[u] = there && norm ? wn[static_cast<size_t>(i0 + u) * a.heads * a.dim] : 0.f;
      }
#pragma unroll
      for (int u = 0; u < kAhead; ++u) {
        if (i0 + u >= stop) break;
        const float f = !GATED ? constant : i0 + u < pieces - 1 ? s_f[i0 + u - base] : 0.f;
        if (mine) w[(i0 + u) * stride] = run;
        run = make_float4(fmaf(run.x, f, own[u].x), fmaf(run.y, f, own[u].y), fmaf(run.z, f, own[u].z), fmaf(run.w, f, own[u].w));
        if (norm) wn[static_cast<size_t>(i0 + u) * a.heads * a.dim] = run_n;
        run_n = fmaf(run_n, f, own_n[u]);
      }
    }
  }
}

// ---- matrix memory ---------------------------------------------------------------------------------------------------
struct Gates {
  const float* logits;          // [rows, stride]: input gates of all heads, then forget gates
  long long stride;
  const float* in_bias;
  const float* forget_bias;
  float cap;
};

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ void log_gates(const Gates& g, int row, int heads, int h, float* in, float* forget) {
  const float* z = g.logits + static_cast<long long>(row) * g.stride;
  *in = g.cap * tanhf((z[h] + g.in_bias[h]) / g.cap);
  *forget = log_sigmoid(g.cap * tanhf((z[heads + h] + g.forget_bias[h]) / g.cap));
}

// One block per (sequence, head), 1024 tokens at a time. m_t = max(m_(t-1) + f_t, i_t) is a scan of pairs
// (sum of f, maximum): (F1, M1) before (F2, M2) gives (F1 + F2, max(M1 + F2, M2)).
constexpr int kGateThreads = 1024;
__global__ void __launch_bounds__(kGateThreads)
memory_gates_kernel(const Args a, const Gates g, float* __restrict__ log_decay, float* __restrict__ log_take, float* __restrict__ maximum) {
  __shared__ float s_f[32], s_m[32], s_top[kGateThreads + 1];
  const int seg = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row0 = a.cu_rows[seg], row1 = a.cu_rows[seg + 1];
  if (row0 >= row1) return;
  float* slot = slot_maximum(a, seg, h);
  float before = a.positions[row0] == 0 ? 0.f : *slot;
  for (int base = row0; base < row1; base += kGateThreads) {
    const int row = base + threadIdx.x;
    float in = -INFINITY, forget = 0.f;
    if (row < row1) log_gates(g, row, a.heads, h, &in, &forget);
    auto scan = [&](float& f, float& m) {   // inclusive, over a warp
#pragma unroll
      for (int off = 1; off < 32; off <<= 1) {
        const float fu = __shfl_up_sync(0xffffffffu, f, off), mu = __shfl_up_sync(0xffffffffu, m, off);
        if (lane >= off) { m = fmaxf(mu + f, m); f += fu; }
      }
    };
    float f = forget, m = in;
    scan(f, m);
    if (lane == 31) { s_f[warp] = f; s_m[warp] = m; }
    __syncthreads();
    if (warp == 0) {
      float wf = s_f[lane], wm = s_m[lane];
      scan(wf, wm);
      s_f[lane] = wf;
      s_m[lane] = wm;
    }
    __syncthreads();
    const float ahead = warp == 0 ? before : fmaxf(before + s_f[warp - 1], s_m[warp - 1]);      // of this warp's tokens
    const float top = fmaxf(ahead + f, m);
    s_top[threadIdx.x + 1] = top;
    if (threadIdx.x == 0) s_top[0] = before;
    __syncthreads();
    if (row < row1) {
      const size_t at = static_cast<size_t>(row) * a.heads + h;
      log_decay[at] = forget + s_top[threadIdx.x] - top;
      log_take[at] = in - top;
      maximum[at] = top;
    }
    before = s_top[min(row1 - base, kGateThreads)];
    __syncthreads();
  }
  if (threadIdx.x == 0) *slot = before;
}

// What a head's sums become: o over max(|q . n|, exp(-m)) + 1e-6.
__device__ __forceinline__ float over_normaliser(float nq, float m) { return 1.f / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f); }

// out = o / rms(o) * weight * sigmoid(gate), a warp per (row, head); o is first divided by its normaliser
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
memory_norm_kernel(const T* __restrict__ o, const float* __restrict__ normaliser, const float* __restrict__ maximum, const T* __restrict__ gate,
                   long long gate_stride, const float* __restrict__ w, float eps, T* __restrict__ out, int units, int heads, int vdim) {
  const int unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= units) return;
  const int row = unit / heads, h = unit % heads;
  const float by = over_normaliser(normaliser[unit], maximum[unit]);
  const T* src = o + static_cast<size_t>(unit) * vdim;
  const T* gsrc = gate + static_cast<size_t>(row) * gate_stride + static_cast<size_t>(h) * vdim;
  const float* wsrc = w + static_cast<size_t>(h) * vdim;
  T* dst = out + static_cast<size_t>(unit) * vdim;
  constexpr int N = 2;                  // pieces per lane that stay in registers, everything requested before the sum
  if (vdim <= 32 * VEC * N) {
    float x[N][VEC], gt[N][VEC], wv[N][VEC], ss = 0.f;
#pragma unroll
    for (int k = 0; k < N; ++k) {
      const int c = (k * 32 + lane) * VEC;
      if (c < vdim) {
        load_vec<T, VEC>(src + c, x[k]);
        load_vec<T, VEC>(gsrc + c, gt[k]);
        load_vec<float, VEC>(wsrc + c, wv[k]);
      }
    }
#pragma unroll
    for (int k = 0; k < N; ++k)
      if ((k * 32 + lane) * VEC < vdim)
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss = fmaf(x[k][i] * by, x[k][i] * by, ss);
    const float inv = by / sqrtf(warp_sum(ss) / static_cast<float>(vdim) + eps);
#pragma unroll
    for (int k = 0; k < N; ++k) {
      const int c = (k * 32 + lane) * VEC;
      if (c < vdim) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[k][i] = x[k][i] * inv * wv[k][i] * sigmoid_exact(gt[k][i]);
        store_vec<T, VEC>(dst + c, x[k]);
      }
    }
    return;
  }
  float ss = 0.f;
  for (int c = lane * VEC; c < vdim; c += 32 * VEC) {
    float x[VEC];
    load_vec<T, VEC>(src + c, x);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(x[i] * by, x[i] * by, ss);
  }
  const float inv = by / sqrtf(warp_sum(ss) / static_cast<float>(vdim) + eps);
  for (int c = lane * VEC; c < vdim; c += 32 * VEC) {
    float x[VEC], gt[VEC], wv[VEC];
    load_vec<T, VEC>(src + c, x);
    load_vec<T, VEC>(gsrc + c, gt);
    load_vec<float, VEC>(wsrc + c, wv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] = x[i] * inv * wv[i] * sigmoid_exact(gt[i]);
    store_vec<T, VEC>(dst + c, x);
  }
}

template <typename T>
__global__ void __launch_bounds__(256, 4)
memory_step_kernel(const Args a, const Gates g, const T* __restrict__ gate, long long gate_stride, const float* __restrict__ w, float eps) {
  __shared__ float4 s_red[256];
  __shared__ float scratch[32];
  extern __shared__ float s_kq[];           // [2][dim]
  const int seg = blockIdx.x, h = blockIdx.y;
  const int row = a.cu_rows[seg];
  const int groups_per_row = a.vdim / 4;                 // float4 columns
  const int lanes_rows = 256 / groups_per_row;           // state rows per pass
  const int cg = threadIdx.x % groups_per_row, rg = threadIdx.x / groups_per_row;
  const bool active = rg < lanes_rows;
  const size_t off = static_cast<size_t>(row) * a.stride;
  const bool fresh = a.positions[row] == 0;
  float4* state = reinterpret_cast<float4*>(slot_state(a, seg, h));
  constexpr int U = 8;                                   // loads in flight per thread
  float4 s[U];
  auto fetch = [&](int d0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int d = d0 + u * lanes_rows;
      s[u] = (d < a.dim && !fresh) ? state[static_cast<size_t>(d) * groups_per_row + cg] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  if (active) fetch(rg);                                 // (the state travels while the gates are worked out)
  float in, forget;
  log_gates(g, row, a.heads, h, &in, &forget);
  float* slot_m = slot_maximum(a, seg, h);
  const float before = fresh ? 0.f : *slot_m;
  const float top = fmaxf(forget + before, in);
  const float decay = fresh ? 0.f : expf(forget + before - top), take = expf(in - top);
  float* slot_n = slot_normaliser(a, seg, h);
  float nq = 0.f;
  for (int d = threadIdx.x; d < a.dim; d += 256) {
    const float k = Elem<T>::ld(static_cast<const T*>(a.k) + off + static_cast<size_t>(h) * a.dim + d) * take;
    const float q = Elem<T>::ld(static_cast<const T*>(a.q) + off + static_cast<size_t>(h) * a.dim + d) * a.q_scale;
    s_kq[d] = k;
    s_kq[a.dim + d] = q;
    const float n = fmaf(fresh ? 0.f : slot_n[d], decay, k);
    slot_n[d] = n;
    nq = fmaf(n, q, nq);
  }
  float v[4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
    v[i] = active ? Elem<T>::ld(static_cast<const T*>(a.v) + off + static_cast<size_t>(h) * a.vdim + cg * 4 + i) : 0.f;
  nq = block_sum_all(nq, scratch);                       // (its barriers also publish s_kq, and everyone has read the maximum)
  if (threadIdx.x == 0) *slot_m = top;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int d0 = rg; active && d0 < a.dim; d0 += U * lanes_rows) {
    if (d0 != rg) fetch(d0);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int d = d0 + u * lanes_rows;
      if (d >= a.dim) break;
      const float k = s_kq[d], q = s_kq[a.dim + d];
      s[u].x = fmaf(s[u].x, decay, k * v[0]); s[u].y = fmaf(s[u].y, decay, k * v[1]);
      s[u].z = fmaf(s[u].z, decay, k * v[2]); s[u].w = fmaf(s[u].w, decay, k * v[3]);
      state[static_cast<size_t>(d) * groups_per_row + cg] = s[u];
      o.x = fmaf(s[u].x, q, o.x); o.y = fmaf(s[u].y, q, o.y); o.z = fmaf(s[u].z, q, o.z); o.w = fmaf(s[u].w, q, o.w);
    }
  }
  s_red[threadIdx.x] = o;
  __syncthreads();
  float ss = 0.f;
  if (rg == 0) {
    for (int r = 1; r < lanes_rows; ++r) {
      const float4 t = s_red[r * groups_per_row + cg];
      o.x += t.x; o.y += t.y; o.z += t.z; o.w += t.w;
    }
    const float by = over_normaliser(nq, top);
    o.x *= by; o.y *= by; o.z *= by; o.w *= by;
    ss = o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w;
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, scratch) / static_cast<float>(a.vdim) + eps);
  if (rg == 0) {
    const size_t col = static_cast<size_t>(h) * a.vdim + cg * 4;
    const T* gt = gate + static_cast<size_t>(row) * gate_stride + col;
    T* dst = static_cast<T*>(a.out) + static_cast<size_t>(row) * a.heads * a.vdim + col;
    const float x[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) Elem<T>::st(dst + i, x[i] * inv * w[col + i] * sigmoid_exact(Elem<T>::ld(gt + i)));
  }
}

// ---- state space -----------------------------------------------------------------------------------------------------
struct Steps {
  const float* z;               // [rows, stride], a column per head
  long long stride;
  const float* bias;
  const float* log_rate;
};
__device__ __forceinline__ void step_gates(const Steps& s, int row, int h, float* dt, float* log_decay) {
  *dt = softplus(s.z[static_cast<long long>(row) * s.stride + h] + s.bias[h]);
  *log_decay = -expf(s.log_rate[h]) * *dt;
}

__global__ void __launch_bounds__(256)
state_space_gates_kernel(const Steps s, int units, int heads, float* __restrict__ log_decay, float* __restrict__ log_take) {
  const int unit = blockIdx.x * 256 + threadIdx.x;
  if (unit >= units) return;
  float dt, decay;
  step_gates(s, unit / heads, unit % heads, &dt, &decay);
  log_decay[unit] = decay;
  log_take[unit] = logf(dt);
}

template <typename T>
__global__ void __launch_bounds__(256, 4)
state_space_step_kernel(const Args a, const Steps s) {
  __shared__ float4 s_red[256];
  extern __shared__ float s_kq[];           // [2][dim]
  const int seg = blockIdx.x, h = blockIdx.y, kh = key_head(a, h);
  const int row = a.cu_rows[seg];
  const int groups_per_row = a.vdim / 4;                 // float4 columns
  const int lanes_rows = 256 / groups_per_row;           // state rows per pass
  const int cg = threadIdx.x % groups_per_row, rg = threadIdx.x / groups_per_row;
  const bool active = rg < lanes_rows;
  const size_t off = static_cast<size_t>(row) * a.stride;
  const bool fresh = a.positions[row] == 0;
  float4* state = reinterpret_cast<float4*>(slot_state(a, seg, h));
  constexpr int U = 8;                                   // loads in flight per thread
  float4 x[U];
  auto fetch = [&](int d0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int d = d0 + u * lanes_rows;
      x[u] = (d < a.dim && !fresh) ? state[static_cast<size_t>(d) * groups_per_row + cg] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  if (active) fetch(rg);                                 // (the state travels while the gates are worked out)
  float dt, decay;
  step_gates(s, row, h, &dt, &decay);
  decay = fresh ? 0.f : expf(decay);
  for (int d = threadIdx.x; d < a.dim; d += 256) {
    s_kq[d] = Elem<T>::ld(static_cast<const T*>(a.k) + off + static_cast<size_t>(kh) * a.dim + d) * dt;
    s_kq[a.dim + d] = Elem<T>::ld(static_cast<const T*>(a.q) + off + static_cast<size_t>(kh) * a.dim + d) * a.q_scale;
  }
  float v[4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
    v[i] = active ? Elem<T>::ld(static_cast<const T*>(a.v) + off + static_cast<size_t>(h) * a.vdim + cg * 4 + i) : 0.f;
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int d0 = rg; active && d0 < a.dim; d0 += U * lanes_rows) {
    if (d0 != rg) fetch(d0);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int d = d0 + u * lanes_rows;
      if (d >= a.dim) break;
      const float k = s_kq[d], q = s_kq[a.dim + d];
      x[u].x = fmaf(x[u].x, decay, k * v[0]); x[u].y = fmaf(x[u].y, decay, k * v[1]);
      x[u].z = fmaf(x[u].z, decay, k * v[2]); x[u].w = fmaf(x[u].w, decay, k * v[3]);
      state[static_cast<size_t>(d) * groups_per_row + cg] = x[u];
      o.x = fmaf(x[u].x, q, o.x); o.y = fmaf(x[u].y, q, o.y); o.z = fmaf(x[u].z, q, o.z); o.w = fmaf(x[u].w, q, o.w);
    }
  }
  s_red[threadIdx.x] = o;
  __syncthreads();
  if (rg == 0) {
    for (int r = 1; r < lanes_rows; ++r) {
      const float4 t = s_red[r * groups_per_row + cg];
      o.x += t.x; o.y += t.y; o.z += t.z; o.w += t.w;
    }
    const float skip = a.skip ? a.skip[h] : 0.f;
    T* dst = static_cast<T*>(a.out) + (static_cast<size_t>(row) * a.heads + h) * a.vdim + cg * 4;
    const float y[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) Elem<T>::st(dst + i, fmaf(skip, v[i], y[i]));
  }
}

bool recurrence_args_ok(const Args& a) {
  return a.positions && a.cu_rows && a.slots && a.q && a.k && a.v && a.state && a.out &&
         a.slot_stride >= static_cast<long long>(a.heads) * a.dim * a.vdim + (a.normaliser ? static_cast<long long>(a.heads) * (a.dim + 1) : 0) && a.segments > 0 && a.heads > 0 &&
         a.heads <= 65535 && a.dim > 0 && a.vdim > 0 && a.num_slots > 0 && a.key_heads >= 0 && (a.key_heads == 0 || a.heads % a.key_heads == 0);
}
bool memory_slots_ok(const Args& a) {        // normalisers and maxima behind the state
  return a.slot_stride >= static_cast<long long>(a.heads) * a.dim * a.vdim + static_cast<long long>(a.heads) * (a.dim + 1);
}

size_t chunk_smem(int dim, int tiles, bool ahead) {
  const int buffers = ahead ? 2 : 1, pitch_v = tiles * 8 + 8;
  return (static_cast<size_t>(2) * buffers * kChunk * (dim + 8) + static_cast<size_t>(buffers + 2) * kChunk * pitch_v + static_cast<size_t>(2) * dim * pitch_v) * 2;
}

// Heads and value columns alone keep the machine busy (two CTAs on most SMs): every sequence in one go.
bool whole_sequences(int heads, int vdim) { return static_cast<long long>(heads) * ((vdim + 8 * kNarrow - 1) / (8 * kNarrow)) >= kNumSMs * 3 / 2; }

// Shorter pieces while all of them still run at once.
int choose_piece(int rows, int segments, int heads, int vdim) {
  int piece = kPiece;
  const long long per_item = static_cast<long long>(heads) * ((vdim + 8 * kWide - 1) / (8 * kWide));
  while (rows > kPiece && piece > kChunk && per_item * ragged_items(rows, segments, piece / 2) <= 2 * kNumSMs) piece /= 2;
  return piece;
}

template <int MT, int NC, bool LOCAL, bool GATED, bool AHEAD>
int launch_chunk(const Args& a, const PieceSpace& ws, int piece, cudaStream_t st) {
  auto kern = recurrence_chunk_kernel<MT, NC, LOCAL, GATED, AHEAD>;
  const size_t smem = chunk_smem(a.dim, NC, AHEAD);
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(ragged_items(a.rows, a.segments, piece), a.heads, (a.vdim + NC * 8 - 1) / (NC * 8)), 128, smem, st>>>(a, ws, piece);
  return launch_status();
}

template <bool GATED>
int launch_passes(const Args& a, float* workspace, bool pieces, cudaStream_t st) {
  if (whole_sequences(a.heads, a.vdim)) {
    constexpr int kAll = 1 << 30;
    const PieceSpace none{};
    return a.dim <= 64 ? launch_chunk<1, kNarrow, false, GATED, true>(a, none, kAll, st) : launch_chunk<2, kNarrow, false, GATED, true>(a, none, kAll, st);
  }
  const int piece = choose_piece(a.rows, a.segments, a.heads, a.vdim);
  const PieceSpace ws = piece_space(a, workspace, ragged_items(a.rows, a.segments, piece));
  if (pieces) {
    const int rc = a.dim <= 64 ? launch_chunk<1, kWide, true, GATED, false>(a, ws, piece, st) : launch_chunk<2, kWide, true, GATED, false>(a, ws, piece, st);
    if (rc != 0) return rc;
    const int z = (a.dim * a.vdim + 1023) / 1024;
    recurrence_scan_kernel<GATED><<<dim3(a.segments, a.heads, z), 256, 0, st>>>(a, ws, piece);
  }
  return a.dim <= 64 ? launch_chunk<1, kWide, false, GATED, false>(a, ws, piece, st) : launch_chunk<2, kWide, false, GATED, false>(a, ws, piece, st);
}

template <typename T, bool GATED>
int launch_simple(const Args& a, cudaStream_t st) {
  const size_t smem = (static_cast<size_t>(a.dim) * 35 + 256 + 32) * 4;
  if (smem > 200 * 1024) return CACHEIR_B200_ELIMIT;
  const dim3 grid(a.segments, a.heads, (a.vdim + 31) / 32);
  cudaError_t e = cudaFuncSetAttribute(recurrence_simple_kernel<T, GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  recurrence_simple_kernel<T, GATED><<<grid, 256, smem, st>>>(a);
  return launch_status();
}

bool decay_ok(const Args& a) { return a.decay_pow || (a.log_decay && a.log_take); }
bool gates_ok(const Gates& g, int heads) { return g.logits && g.in_bias && g.forget_bias && g.cap > 0.f && g.stride >= 2ll * heads; }

}  // namespace
}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_recurrence_simple(const cacheir_b200_recurrence_args* a, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (!recurrence_args_ok(*a)) return CACHEIR_B200_EINVAL;
  if (!decay_ok(*a)) return CACHEIR_B200_EINVAL;
  CB200_HYBRID_DTYPE(a->dtype, return a->decay_pow ? launch_simple<T, false>(*a, as_stream(stream)) : launch_simple<T, true>(*a, as_stream(stream)));
  return CACHEIR_B200_EUNSUPPORTED;
}

extern "C" int cacheir_b200_recurrence_step(const cacheir_b200_recurrence_args* a, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (!recurrence_args_ok(*a) || !a->decay_pow || a->key_heads != 0 || a->skip || a->rows != a->segments) return CACHEIR_B200_EINVAL;
  if (a->vdim % 4 != 0 || a->vdim > 1024 || a->dim > 4096) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(a->state, 16) || a->slot_stride % 4 != 0) return CACHEIR_B200_EALIGN;
  const dim3 grid(a->segments, a->heads);
  const size_t smem = static_cast<size_t>(a->dim) * 8;
  if (a->dtype == CACHEIR_B200_F32) recurrence_step_kernel<float><<<grid, 256, smem, as_stream(stream)>>>(*a);
  else if (a->dtype == CACHEIR_B200_BF16) recurrence_step_kernel<__nv_bfloat16><<<grid, 256, smem, as_stream(stream)>>>(*a);
  else return CACHEIR_B200_EUNSUPPORTED;
  return launch_status();
}

extern "C" int cacheir_b200_recurrence_chunked_supported(int dim, int vdim, int dtype) {
  return dtype == CACHEIR_B200_BF16 && dim >= 16 && dim % 16 == 0 && dim <= 128 && vdim % 8 == 0 ? 1 : 0;
}

extern "C" size_t cacheir_b200_recurrence_workspace_bytes(int rows, int segments, int heads, int dim, int vdim) {
  if (rows <= kPiece || whole_sequences(heads, vdim)) return 0;
  return static_cast<size_t>(ragged_items(rows, segments, choose_piece(rows, segments, heads, vdim))) * heads * (static_cast<size_t>(dim) * (vdim + 1) + 1) * 4;
}

extern "C" int cacheir_b200_recurrence_chunked(const cacheir_b200_recurrence_args* a, void* workspace, size_t workspace_bytes, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (!recurrence_args_ok(*a) || !decay_ok(*a)) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_recurrence_chunked_supported(a->dim, a->vdim, a->dtype)) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(a->q, 16) || !aligned_to(a->k, 16) || !aligned_to(a->v, 16) || !aligned_to(a->out, 16) || a->stride % 8 != 0 ||
      !aligned_to(a->state, 16) || a->slot_stride % 4 != 0)
    return CACHEIR_B200_EALIGN;
  const size_t need = cacheir_b200_recurrence_workspace_bytes(a->rows, a->segments, a->heads, a->dim, a->vdim);
  if (need > 0 && (!workspace || workspace_bytes < need)) return CACHEIR_B200_EWORKSPACE;
  float* ws = static_cast<float*>(workspace);
  return a->decay_pow ? launch_passes<false>(*a, ws, need > 0, as_stream(stream)) : launch_passes<true>(*a, ws, need > 0, as_stream(stream));
}

extern "C" int cacheir_b200_memory_gates(const cacheir_b200_recurrence_args* a, const float* logits, long long stride, const float* in_bias,
                                         const float* forget_bias, float cap, float* log_decay, float* log_take, float* maximum, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  const Gates g{logits, stride, in_bias, forget_bias, cap};
  if (!recurrence_args_ok(*a) || !memory_slots_ok(*a) || a->decay_pow || !gates_ok(g, a->heads) || !log_decay || !log_take || !maximum) return CACHEIR_B200_EINVAL;
  memory_gates_kernel<<<dim3(a->segments, a->heads), kGateThreads, 0, as_stream(stream)>>>(*a, g, log_decay, log_take, maximum);
  return launch_status();
}

extern "C" int cacheir_b200_memory_norm(const void* o, const float* normaliser, const float* maximum, const void* gate, long long gate_stride,
                                        const float* w, float eps, void* out, int rows, int heads, int vdim, int dtype, void* stream) {
  if (rows <= 0) return 0;
  if (!o || !normaliser || !maximum || !gate || !w || !out || heads <= 0 || vdim <= 0) return CACHEIR_B200_EINVAL;
  const int quad = 4 * (dtype == CACHEIR_B200_F32 ? 4 : 2), units = rows * heads;
  const bool vec = vdim % 4 == 0 && gate_stride % 4 == 0 && aligned_to(o, quad) && aligned_to(gate, quad) && aligned_to(w, 16) && aligned_to(out, quad);
  const int grid = (units + 7) / 8;
#define CB200_NORM(VEC)                                                                                                              \
  memory_norm_kernel<T, VEC><<<grid, 256, 0, as_stream(stream)>>>(static_cast<const T*>(o), normaliser, maximum, static_cast<const T*>(gate), \
                                                                 gate_stride, w, eps, static_cast<T*>(out), units, heads, vdim)
  CB200_HYBRID_DTYPE(dtype, {
    if (vec) CB200_NORM(4);
    else CB200_NORM(1);
  });
#undef CB200_NORM
  return launch_status();
}

extern "C" int cacheir_b200_memory_step(const cacheir_b200_recurrence_args* a, const float* logits, long long stride, const float* in_bias,
                                        const float* forget_bias, float cap, const void* gate, long long gate_stride, const float* w, float eps,
                                        void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  const Gates g{logits, stride, in_bias, forget_bias, cap};
  if (!recurrence_args_ok(*a) || !memory_slots_ok(*a) || a->decay_pow || a->key_heads != 0 || a->skip || !gates_ok(g, a->heads) || !gate || !w ||
      a->rows != a->segments)
    return CACHEIR_B200_EINVAL;
  if (a->vdim % 4 != 0 || a->vdim > 1024 || a->dim > 4096) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(a->state, 16) || a->slot_stride % 4 != 0) return CACHEIR_B200_EALIGN;
  const dim3 grid(a->segments, a->heads);
  const size_t smem = static_cast<size_t>(a->dim) * 8;
  CB200_HYBRID_DTYPE(a->dtype, (memory_step_kernel<T><<<grid, 256, smem, as_stream(stream)>>>(*a, g, static_cast<const T*>(gate), gate_stride, w, eps)));
  return launch_status();
}

extern "C" int cacheir_b200_state_space_gates(const cacheir_b200_recurrence_args* a, const float* z, long long stride, const float* bias,
                                              const float* log_rate, float* log_decay, float* log_take, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (a->heads <= 0 || !z || stride < a->heads || !bias || !log_rate || !log_decay || !log_take) return CACHEIR_B200_EINVAL;
  const int units = a->rows * a->heads;
  state_space_gates_kernel<<<(units + 255) / 256, 256, 0, as_stream(stream)>>>(Steps{z, stride, bias, log_rate}, units, a->heads, log_decay, log_take);
  return launch_status();
}

extern "C" int cacheir_b200_state_space_step(const cacheir_b200_recurrence_args* a, const float* z, long long stride, const float* bias,
                                             const float* log_rate, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (!recurrence_args_ok(*a) || a->decay_pow || a->rows != a->segments || !z || stride < a->heads || !bias || !log_rate) return CACHEIR_B200_EINVAL;
  if (a->vdim % 4 != 0 || a->vdim > 1024 || a->dim > 4096) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(a->state, 16) || a->slot_stride % 4 != 0) return CACHEIR_B200_EALIGN;
  const size_t smem = static_cast<size_t>(a->dim) * 8;
  CB200_HYBRID_DTYPE(a->dtype, (state_space_step_kernel<T><<<dim3(a->segments, a->heads), 256, smem, as_stream(stream)>>>(*a, Steps{z, stride, bias, log_rate})));
  return launch_status();
}

extern "C" int cacheir_b200_recurrence_device_status(int) { return 0; }
