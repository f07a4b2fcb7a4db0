// Linear recurrence S <- decay S + k v^T, o = S^T q per head, float32 state carried per sequence slot, sm_100a.
//
// simple   any extents and types: one CTA per (sequence, head, 32 value columns) walks the tokens, state in shared memory
// step     decode: one CTA per (sequence, head) streams the state once (16-byte accesses), HBM bound
// chunked  prompts, bf16 operands on the tensor cores, 64 tokens at a time. With D_ij = decay^(i-j) for j <= i:
//            O = diag(decay^(i+1)) Q S + ((Q K^T) o D) V        S' = decay^n S + K^T diag(decay^(n-1-j)) V
//          The state stays in float32 registers; whatever is float32 by nature and has to enter an MMA (the state, the
//          decayed scores, the decayed values) goes in as a sum of two bf16 numbers. Sequences are cut into 256-token
//          pieces that run in parallel: a first pass finds every piece's own contribution, a scan turns these into the
//          pieces' initial states, and the main pass starts from them.
#include "cacheir_b200_hybrid.h"
#include "hybrid_common.cuh"
#include "ragged.cuh"

namespace cb200 {
namespace {

constexpr int kPowers = 65;
constexpr int kChunk = 64;
constexpr int kPiece = 256;
constexpr int kCols = 64;          // value columns per CTA of the chunked form
constexpr int kPitchV = kCols + 8; // bf16 elements per shared-memory row (16 bytes over a multiple of 128: conflict-free)

using Args = cacheir_b200_recurrence_args;

__device__ __forceinline__ float* slot_state(const Args& a, int seg, int h) {
  const int slot = min(max(a.slots[seg], 0), a.num_slots - 1);
  return a.state + (static_cast<size_t>(slot) * a.heads + h) * a.dim * a.vdim;
}

template <typename T>
__global__ void __launch_bounds__(256)
recurrence_simple_kernel(const Args a) {
  extern __shared__ float sm[];
  float* s_state = sm;                       // [dim][32]
  float* s_k = s_state + a.dim * 32;         // [dim]
  float* s_q = s_k + a.dim;                  // [dim]
  float* s_red = s_q + a.dim;                // [8][32]
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
  const float decay = a.decay_pow[h * kPowers + 1];
  for (int row = row0; row < row1; ++row) {
    __syncthreads();
    const size_t off = static_cast<size_t>(row) * a.stride;
    for (int d = threadIdx.x; d < a.dim; d += 256) {
      s_k[d] = Elem<T>::ld(static_cast<const T*>(a.k) + off + static_cast<size_t>(h) * a.dim + d);
      s_q[d] = Elem<T>::ld(static_cast<const T*>(a.q) + off + static_cast<size_t>(h) * a.dim + d);
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
      float t = 0.f;
#pragma unroll
      for (int g = 0; g < 8; ++g) t += s_red[g * 32 + lane];
      Elem<T>::st(static_cast<T*>(a.out) + (static_cast<size_t>(row) * a.heads + h) * a.vdim + col, t);
    }
  }
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
// MT = 16-row state tiles per warp (dim <= 64 MT)
template <int MT, bool LOCAL>
__global__ void __launch_bounds__(128)
recurrence_chunk_kernel(const Args a, float* __restrict__ ws) {
  extern __shared__ __align__(16) uint8_t raw[];
  const int dim = a.dim;
  const int pitch = dim + 8;
  __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(raw);        // [64][pitch]
  __nv_bfloat16* s_k = s_q + kChunk * pitch;                         // [64][pitch]
  __nv_bfloat16* s_v = s_k + kChunk * pitch;                         // [64][72]
  __nv_bfloat16* s_dv = s_v + kChunk * kPitchV;                      // [2][64][72] decayed values, hi | lo
  __nv_bfloat16* s_s = s_dv + 2 * kChunk * kPitchV;                  // [2][dim][72] state, hi | lo
  __shared__ float s_pow[kPowers];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, v0 = blockIdx.z * kCols;

  const RaggedItem it = find_item(a.cu_rows, a.segments, kPiece, blockIdx.x);
  if (it.seg < 0) return;
  const bool alone = it.last && static_cast<int>(blockIdx.x) == it.first;     // the segment is a single piece
  if (LOCAL && it.last) return;                                               // nobody needs its contribution
  for (int i = threadIdx.x; i < kPowers; i += 128) s_pow[i] = a.decay_pow[h * kPowers + i];

  float st[MT][8][4];          // state rows (warp + 4 t)*16 .. +15, columns v0 .. v0+63
  float* state = slot_state(a, it.seg, h);
  float* piece = ws + (static_cast<size_t>(blockIdx.x) * a.heads + h) * dim * a.vdim;
  const float* init = alone ? state : piece;
  const bool zero = LOCAL || (alone && a.positions[it.row0] == 0);
  const int cols = min(kCols, a.vdim - v0);
#pragma unroll
  for (int t = 0; t < MT; ++t)
#pragma unroll
    for (int n = 0; n < 8; ++n)
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
  for (int r0 = 0; r0 < it.count; r0 += kChunk) {
    const int n = min(kChunk, it.count - r0);
    const size_t base = static_cast<size_t>(it.row0 + r0);
    for (int i = threadIdx.x; i < kChunk * kc; i += 128) {
      const int r = i / kc, c = i % kc;
      uint4 q = make_uint4(0u, 0u, 0u, 0u), k = q;
      if (r < n) {
        const size_t off = (base + r) * a.stride + static_cast<size_t>(h) * dim + c * 8;
        if (!LOCAL) q = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.q) + off);
        k = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.k) + off);
      }
      if (!LOCAL) *reinterpret_cast<uint4*>(s_q + r * pitch + c * 8) = q;
      *reinterpret_cast<uint4*>(s_k + r * pitch + c * 8) = k;
    }
    for (int i = threadIdx.x; i < kChunk * (kCols / 8); i += 128) {
      const int r = i / (kCols / 8), c = i % (kCols / 8);
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < n && c * 8 < cols)
        v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.v) + (base + r) * a.stride + static_cast<size_t>(h) * a.vdim + v0 + c * 8);
      if (!LOCAL) *reinterpret_cast<uint4*>(s_v + r * kPitchV + c * 8) = v;
      const float f = s_pow[max(n - 1 - r, 0)];
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
        for (int nn = 0; nn < 8; ++nn)
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

    if (!LOCAL && warp * 16 < n) {
      float o[8][4];
#pragma unroll
      for (int nn = 0; nn < 8; ++nn)
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
          for (int nn = 0; nn < 8; nn += 2) {
            uint32_t bf[4];
            ldsm_x4_t(sa + ((part * dim + k * 16) * kPitchV + nn * 8) * 2, bf);
            mma_bf16(o[nn], af, bf[0], bf[1]);
            mma_bf16(o[nn + 1], af, bf[2], bf[3]);
          }
      }
      const int i0 = warp * 16 + (lane >> 2);
      const float f0 = s_pow[i0 + 1], f1 = s_pow[i0 + 9];
#pragma unroll
      for (int nn = 0; nn < 8; ++nn) {
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
            d[u][e] = j <= i ? sc[2 * kk + u][e] * s_pow[i - j] : 0.f;
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
        for (int nn = 0; nn < 8; nn += 2) {
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
        if (i < n) {
          __nv_bfloat16* dst = out + ((base + i) * a.heads + h) * a.vdim + v0;
#pragma unroll
          for (int nn = 0; nn < 8; ++nn) {
            const int c = nn * 8 + (lane & 3) * 2;
            if (c < cols) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(o[nn][e * 2], o[nn][e * 2 + 1]);
          }
        }
      }
    }

    // S' = decay^n S + K^T (decayed V)
    const float fn = s_pow[n];
    const uint32_t kt = smem_addr(s_k) + (((lane & 7) + ((lane >> 4) & 1) * 8) * pitch + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t dv = smem_addr(s_dv) + (((lane & 7) + ((lane >> 3) & 1) * 8) * kPitchV + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      const int m0 = (warp + 4 * t) * 16;
      if (m0 >= dim) continue;
#pragma unroll
      for (int nn = 0; nn < 8; ++nn)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[t][nn][e] *= fn;
#pragma unroll
      for (int k = 0; k < kChunk / 16; ++k) {
        uint32_t af[4];
        ldsm_x4_t(kt + (k * 16 * pitch + m0) * 2, af);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int nn = 0; nn < 8; nn += 2) {
            uint32_t bf[4];
            ldsm_x4_t(dv + ((part * kChunk + k * 16) * kPitchV + nn * 8) * 2, bf);
            mma_bf16(st[t][nn], af, bf[0], bf[1]);
            mma_bf16(st[t][nn + 1], af, bf[2], bf[3]);
          }
      }
    }
    __syncthreads();
  }

  float* dst = LOCAL ? piece : state;
  if (LOCAL || it.last) {
#pragma unroll
    for (int t = 0; t < MT; ++t)
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int d = (warp + 4 * t) * 16 + (lane >> 2) + e * 8, c = n * 8 + (lane & 3) * 2;
          if (d < dim && c < cols)
            *reinterpret_cast<float2*>(dst + static_cast<size_t>(d) * a.vdim + v0 + c) = make_float2(st[t][n][e * 2], st[t][n][e * 2 + 1]);
        }
  }
}

// Contributions of a segment's pieces -> their initial states (in place).
__global__ void __launch_bounds__(256)
recurrence_scan_kernel(const Args a, float* __restrict__ ws) {
  const int seg = blockIdx.x, h = blockIdx.y;
  int first = 0;
  for (int s = 0; s < seg; ++s) first += (a.cu_rows[s + 1] - a.cu_rows[s] + kPiece - 1) / kPiece;
  const int rows = a.cu_rows[seg + 1] - a.cu_rows[seg];
  const int pieces = (rows + kPiece - 1) / kPiece;
  if (pieces < 2) return;
  const size_t plane = static_cast<size_t>(a.dim) * a.vdim;
  const float p64 = a.decay_pow[h * kPowers + 64];
  const float f = (p64 * p64) * (p64 * p64);
  const bool fresh = a.positions[a.cu_rows[seg]] == 0;
  const float* state = slot_state(a, seg, h);
  for (size_t e = static_cast<size_t>(blockIdx.z) * 256 + threadIdx.x; e < plane; e += static_cast<size_t>(gridDim.z) * 256) {
    float run = fresh ? 0.f : state[e];
    for (int i = 0; i < pieces; ++i) {
      float* w = ws + (static_cast<size_t>(first + i) * a.heads + h) * plane + e;
      const float own = i + 1 < pieces ? *w : 0.f;
      *w = run;
      run = fmaf(run, f, own);
    }
  }
}

bool recurrence_args_ok(const Args& a) {
  return a.positions && a.cu_rows && a.slots && a.q && a.k && a.v && a.decay_pow && a.state && a.out && a.segments > 0 && a.heads > 0 &&
         a.heads <= 65535 && a.dim > 0 && a.vdim > 0 && a.num_slots > 0;
}

size_t chunk_smem(int dim) {
  return (static_cast<size_t>(2) * kChunk * (dim + 8) + static_cast<size_t>(3) * kChunk * kPitchV + static_cast<size_t>(2) * dim * kPitchV) * 2;
}

template <int MT, bool LOCAL>
int launch_chunk(const Args& a, float* ws, cudaStream_t st) {
  auto kern = recurrence_chunk_kernel<MT, LOCAL>;
  const size_t smem = chunk_smem(a.dim);
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(ragged_items(a.rows, a.segments, kPiece), a.heads, (a.vdim + kCols - 1) / kCols), 128, smem, st>>>(a, ws);
  return launch_status();
}

}  // namespace
}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_recurrence_simple(const cacheir_b200_recurrence_args* a, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (!recurrence_args_ok(*a)) return CACHEIR_B200_EINVAL;
  const size_t smem = (static_cast<size_t>(a->dim) * 34 + 256) * 4;
  if (smem > 200 * 1024) return CACHEIR_B200_ELIMIT;
  const dim3 grid(a->segments, a->heads, (a->vdim + 31) / 32);
  cudaStream_t st = as_stream(stream);
  if (a->dtype == CACHEIR_B200_F32) {
    cudaFuncSetAttribute(recurrence_simple_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    recurrence_simple_kernel<float><<<grid, 256, smem, st>>>(*a);
  } else if (a->dtype == CACHEIR_B200_BF16) {
    cudaFuncSetAttribute(recurrence_simple_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    recurrence_simple_kernel<__nv_bfloat16><<<grid, 256, smem, st>>>(*a);
  } else {
    return CACHEIR_B200_EUNSUPPORTED;
  }
  return launch_status();
}

extern "C" int cacheir_b200_recurrence_step(const cacheir_b200_recurrence_args* a, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (!recurrence_args_ok(*a) || a->rows != a->segments) return CACHEIR_B200_EINVAL;
  if (a->vdim % 4 != 0 || a->vdim > 1024 || a->dim > 4096) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(a->state, 16)) return CACHEIR_B200_EALIGN;
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
  if (rows <= kPiece) return 0;
  return static_cast<size_t>(ragged_items(rows, segments, kPiece)) * heads * dim * vdim * 4;
}

extern "C" int cacheir_b200_recurrence_chunked(const cacheir_b200_recurrence_args* a, void* workspace, size_t workspace_bytes, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (!recurrence_args_ok(*a)) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_recurrence_chunked_supported(a->dim, a->vdim, a->dtype)) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(a->q, 16) || !aligned_to(a->k, 16) || !aligned_to(a->v, 16) || !aligned_to(a->out, 16) || a->stride % 8 != 0 ||
      !aligned_to(a->state, 16))
    return CACHEIR_B200_EALIGN;
  const size_t need = cacheir_b200_recurrence_workspace_bytes(a->rows, a->segments, a->heads, a->dim, a->vdim);
  if (need > 0 && (!workspace || workspace_bytes < need)) return CACHEIR_B200_EWORKSPACE;
  cudaStream_t st = as_stream(stream);
  float* ws = static_cast<float*>(workspace);
  if (need > 0) {
    const int rc = a->dim <= 64 ? launch_chunk<1, true>(*a, ws, st) : launch_chunk<2, true>(*a, ws, st);
    if (rc != 0) return rc;
    const int z = (a->dim * a->vdim + 1023) / 1024;
    recurrence_scan_kernel<<<dim3(a->segments, a->heads, z), 256, 0, st>>>(*a, ws);
  }
  return a->dim <= 64 ? launch_chunk<1, false>(*a, ws, st) : launch_chunk<2, false>(*a, ws, st);
}
