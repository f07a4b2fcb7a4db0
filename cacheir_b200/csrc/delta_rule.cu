// Gated delta rule S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q per head, float32 state carried per sequence slot,
// sm_100a. Rows of q and k come as the convolution left them; their lengths are divided out here, in float32.
//
// simple   any extents and types: one CTA per (sequence, head, 32 value columns) walks the tokens, state in shared memory
// step     decode: one CTA per (sequence, head). S^T k and S^T q come out of one pass over the state, o = g S^T q + (k . q) u,
//          and the state is written back from registers; the head's norm and the output gate follow.
// chunked  prompts, 64 tokens at a time. With c the running sum of log decays in a chunk and A the strictly lower triangle of
//          beta_i exp(c_i - c_j) k_i . k_j, the chunk's writes are U = M beta (V - exp(c) K S), M = (I + A)^-1, and
//            O = exp(c) Q S + P U,  P_ij = exp(c_i - c_j) q_i . k_j (j <= i),     S' = exp(c_n) S + K^T (exp(c_n - c_j) U)
//          local  M and P of every chunk and head, in parallel: products on the tensor cores, the inverse in float32 (diagonal
//                 blocks of 16 by substitution, then doubled twice)
//          chain  one CTA per (sequence, head, 32 or 16 value columns) runs through the chunks, state in float32 registers
//          Whatever is float32 by nature and has to enter an MMA goes in as a sum of two bf16 numbers.
#include "cacheir_b200_delta.h"
#include "hybrid_common.cuh"
#include "ragged.cuh"

namespace cb200 {
namespace {

using Args = cacheir_b200_delta_args;
constexpr float kUnitEps = 1e-6f;
constexpr int kChunk = 64;

__device__ __forceinline__ float* slot_state(const Args& a, int seg, int h) {
  const int slot = min(max(a.slots[seg], 0), a.num_slots - 1);
  return a.state + static_cast<size_t>(slot) * a.slot_stride + static_cast<size_t>(h) * a.dim * a.vdim;
}
__device__ __forceinline__ int key_head(const Args& a, int h) { return h / (a.heads / a.key_heads); }
__device__ __forceinline__ void delta_gates(const Args& a, size_t row, int h, float* beta, float* log_decay) {
  const float* z = a.z + row * a.z_stride;
  *beta = 1.f / (1.f + expf(-z[h]));
  *log_decay = -expf(a.log_rate[h]) * softplus(z[a.heads + h] + a.bias[h]);
}

template <typename T>
__global__ void __launch_bounds__(256)
delta_simple_kernel(const Args a) {
  extern __shared__ float sm[];
  float* s_state = sm;                       // [dim][32]
  float* s_k = s_state + a.dim * 32;         // [dim]
  float* s_q = s_k + a.dim;                  // [dim]
  float* s_red = s_q + a.dim;                // [2][8][32]
  float* s_sum = s_red + 512;                // [32]
  const int seg = blockIdx.x, h = blockIdx.y, kh = key_head(a, h);
  const int row0 = a.cu_rows[seg], row1 = a.cu_rows[seg + 1];
  if (row0 >= row1) return;
  const int lane = threadIdx.x & 31, group = threadIdx.x >> 5;
  const int col = blockIdx.z * 32 + lane;
  const bool col_ok = col < a.vdim;
  float* state = slot_state(a, seg, h);
  const bool fresh = a.positions[row0] == 0;
  for (int d = group; d < a.dim; d += 8)
    s_state[d * 32 + lane] = (fresh || !col_ok) ? 0.f : state[static_cast<size_t>(d) * a.vdim + col];
  const float q_scale = 1.f / sqrtf(static_cast<float>(a.dim));
  for (int row = row0; row < row1; ++row) {
    __syncthreads();
    const size_t off = static_cast<size_t>(row) * a.stride;
    float kk = 0.f, qq = 0.f;
    for (int d = threadIdx.x; d < a.dim; d += 256) {
      const float k = Elem<T>::ld(static_cast<const T*>(a.k) + off + static_cast<size_t>(kh) * a.dim + d);
      const float q = Elem<T>::ld(static_cast<const T*>(a.q) + off + static_cast<size_t>(kh) * a.dim + d);
      s_k[d] = k;
      s_q[d] = q;
      kk = fmaf(k, k, kk);
      qq = fmaf(q, q, qq);
    }
    const float nk = 1.f / sqrtf(block_sum_all(kk, s_sum) + kUnitEps), nq = q_scale / sqrtf(block_sum_all(qq, s_sum) + kUnitEps);
    float beta, log_decay;
    delta_gates(a, row, h, &beta, &log_decay);
    const float decay = expf(log_decay);
    const float v = col_ok ? Elem<T>::ld(static_cast<const T*>(a.v) + off + static_cast<size_t>(h) * a.vdim + col) : 0.f;
    float met = 0.f;
    for (int d = group; d < a.dim; d += 8) {
      const float s = s_state[d * 32 + lane] * decay;
      s_state[d * 32 + lane] = s;
      met = fmaf(s, s_k[d] * nk, met);
    }
    s_red[group * 32 + lane] = met;
    __syncthreads();
    met = 0.f;
#pragma unroll
    for (int g = 0; g < 8; ++g) met += s_red[g * 32 + lane];
    const float u = beta * (v - met);
    float o = 0.f;
    for (int d = group; d < a.dim; d += 8) {
      const float s = fmaf(s_k[d] * nk, u, s_state[d * 32 + lane]);
      s_state[d * 32 + lane] = s;
      o = fmaf(s, s_q[d] * nq, o);
    }
    s_red[256 + group * 32 + lane] = o;
    __syncthreads();
    if (group == 0 && col_ok) {
      float t = 0.f;
#pragma unroll
      for (int g = 0; g < 8; ++g) t += s_red[256 + g * 32 + lane];
      Elem<T>::st(static_cast<T*>(a.out) + (static_cast<size_t>(row) * a.heads + h) * a.vdim + col, t);
    }
  }
  if (col_ok)
    for (int d = group; d < a.dim; d += 8) state[static_cast<size_t>(d) * a.vdim + col] = s_state[d * 32 + lane];
}

// ---- decoding --------------------------------------------------------------------------------------------------------
// A thread has float4 columns cg of rows rg, rg + lanes, ...; HELD of them stay in registers, further ones are read twice.
template <typename T, int THREADS, int HELD>
__global__ void __launch_bounds__(THREADS)
delta_step_kernel(const Args a, const T* __restrict__ gate, long long gate_stride, const float* __restrict__ w, float eps) {
  __shared__ float4 s_red[2][THREADS];
  __shared__ float s_sum[32];
  extern __shared__ float s_kq[];           // [2][dim] unit key, unit query
  const int seg = blockIdx.x, h = blockIdx.y, kh = key_head(a, h);
  const int row = a.cu_rows[seg];
  const int per_row = a.vdim / 4, lanes = THREADS / per_row;
  const int cg = threadIdx.x % per_row, rg = threadIdx.x / per_row;
  const bool active = rg < lanes;
  const size_t off = static_cast<size_t>(row) * a.stride;
  const bool fresh = a.positions[row] == 0;
  float4* state = reinterpret_cast<float4*>(slot_state(a, seg, h));
  auto at = [&](int d) { return (d < a.dim && !fresh) ? state[static_cast<size_t>(d) * per_row + cg] : make_float4(0.f, 0.f, 0.f, 0.f); };
  float4 s[HELD];
  if (active) {                             // (the state travels while lengths and gates are worked out)
#pragma unroll
    for (int u = 0; u < HELD; ++u) s[u] = at(rg + u * lanes);
  }
  float kk = 0.f, qq = 0.f, kq = 0.f;
  for (int d = threadIdx.x; d < a.dim; d += THREADS) {
    const float k = Elem<T>::ld(static_cast<const T*>(a.k) + off + static_cast<size_t>(kh) * a.dim + d);
    const float q = Elem<T>::ld(static_cast<const T*>(a.q) + off + static_cast<size_t>(kh) * a.dim + d);
    s_kq[d] = k;
    s_kq[a.dim + d] = q;
    kk = fmaf(k, k, kk);
    qq = fmaf(q, q, qq);
    kq = fmaf(k, q, kq);
  }
  float beta, log_decay;
  delta_gates(a, row, h, &beta, &log_decay);
  const float decay = fresh ? 0.f : expf(log_decay);
  float v[4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
    v[i] = active ? Elem<T>::ld(static_cast<const T*>(a.v) + off + static_cast<size_t>(h) * a.vdim + cg * 4 + i) : 0.f;
  // (the sums' barriers also publish s_kq)
  const float nk = 1.f / sqrtf(block_sum_all(kk, s_sum) + kUnitEps);
  const float nq = 1.f / (sqrtf(block_sum_all(qq, s_sum) + kUnitEps) * sqrtf(static_cast<float>(a.dim)));
  kq = block_sum_all(kq, s_sum) * nk * nq;
  float4 met = make_float4(0.f, 0.f, 0.f, 0.f), out = met;      // S^T k, S^T q, before lengths and decay
  auto meet = [&](const float4& x, int d) {
    const float k = s_kq[d], q = s_kq[a.dim + d];
    met.x = fmaf(x.x, k, met.x); met.y = fmaf(x.y, k, met.y); met.z = fmaf(x.z, k, met.z); met.w = fmaf(x.w, k, met.w);
    out.x = fmaf(x.x, q, out.x); out.y = fmaf(x.y, q, out.y); out.z = fmaf(x.z, q, out.z); out.w = fmaf(x.w, q, out.w);
  };
  if (active) {
#pragma unroll
    for (int u = 0; u < HELD; ++u)
      if (rg + u * lanes < a.dim) meet(s[u], rg + u * lanes);
    for (int d = rg + HELD * lanes; d < a.dim; d += lanes) meet(at(d), d);
  }
  s_red[0][threadIdx.x] = met;
  s_red[1][threadIdx.x] = out;
  __syncthreads();
  if (rg == 0) {
    for (int r = 1; r < lanes; ++r) {
      const float4 m = s_red[0][r * per_row + cg], t = s_red[1][r * per_row + cg];
      met.x += m.x; met.y += m.y; met.z += m.z; met.w += m.w;
      out.x += t.x; out.y += t.y; out.z += t.z; out.w += t.w;
    }
    const float f = decay * nk, g = decay * nq;
    met = make_float4(beta * (v[0] - f * met.x), beta * (v[1] - f * met.y), beta * (v[2] - f * met.z), beta * (v[3] - f * met.w));      // u
    out = make_float4(fmaf(kq, met.x, g * out.x), fmaf(kq, met.y, g * out.y), fmaf(kq, met.z, g * out.z), fmaf(kq, met.w, g * out.w));
    s_red[0][cg] = met;                     // (row group 0 alone reads and writes its own first entries)
  }
  __syncthreads();
  if (active) {
    const float4 u4 = s_red[0][cg];
    auto write = [&](float4 x, int d) {
      const float k = s_kq[d] * nk;
      x.x = fmaf(x.x, decay, k * u4.x); x.y = fmaf(x.y, decay, k * u4.y); x.z = fmaf(x.z, decay, k * u4.z); x.w = fmaf(x.w, decay, k * u4.w);
      state[static_cast<size_t>(d) * per_row + cg] = x;
    };
#pragma unroll
    for (int u = 0; u < HELD; ++u)
      if (rg + u * lanes < a.dim) write(s[u], rg + u * lanes);
    for (int d = rg + HELD * lanes; d < a.dim; d += lanes) write(at(d), d);
  }
  const float ss = rg == 0 ? out.x * out.x + out.y * out.y + out.z * out.z + out.w * out.w : 0.f;
  const float inv = 1.f / sqrtf(block_sum_all(ss, s_sum) / static_cast<float>(a.vdim) + eps);
  if (rg == 0) {
    const size_t col = static_cast<size_t>(h) * a.vdim + cg * 4;
    const T* gt = gate + static_cast<size_t>(row) * gate_stride + col;
    T* dst = static_cast<T*>(a.out) + static_cast<size_t>(row) * a.heads * a.vdim + col;
    const float y[4] = {out.x, out.y, out.z, out.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) Elem<T>::st(dst + i, y[i] * inv * w[cg * 4 + i] * silu_exact(Elem<T>::ld(gt + i)));
  }
}

// ---- chunked form ----------------------------------------------------------------------------------------------------
// Between the passes, per (chunk, head): M and P as MMA operands [2][row tile][k tile <= row tile][hi, lo][lane] x 16 bytes, and per
// row log decay sums, beta, and the reciprocal lengths of k and q (the latter with dim^-1/2).
constexpr int kTri = 10;               // 16 x 16 tiles of a lower triangle of four
struct ChunkSpace {
  uint4* tiles;                        // [item][head][2][kTri][2][32]
  float4* rows;                        // [item][head][kChunk]: (c, beta, 1/|k|, dim^-1/2 / |q|)
};
__device__ __forceinline__ uint4* tile_at(const ChunkSpace& ws, size_t unit, int which, int rt, int kt) {
  return ws.tiles + ((unit * 2 + which) * kTri + rt * (rt + 1) / 2 + kt) * 64;
}
__device__ __forceinline__ void split_pair(float x, float y, uint32_t* hi, uint32_t* lo) {
  float h0, l0, h1, l1;
  split_bf16(x, &h0, &l0);
  split_bf16(y, &h1, &l1);
  *hi = pack_bf16(h0, h1);
  *lo = pack_bf16(l0, l1);
}

__global__ void __launch_bounds__(128)
delta_local_kernel(const Args a, const ChunkSpace ws) {
  extern __shared__ __align__(16) uint8_t raw[];
  constexpr int kPitch = kChunk + 4;
  const int dim = a.dim, pitch = dim + 8;
  __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(raw);        // [64][pitch]
  __nv_bfloat16* s_k = s_q + kChunk * pitch;                         // [64][pitch]
  float* s_a = reinterpret_cast<float*>(s_k + kChunk * pitch);       // [64][kPitch] A
  float* s_m = s_a + kChunk * kPitch;                                // [64][kPitch] (I + A)^-1
  float* s_t = s_m + kChunk * kPitch;                                // [32][36]
  __shared__ float4 s_row[kChunk];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, kh = key_head(a, h);
  const RaggedItem it = find_item(a.cu_rows, a.segments, kChunk, blockIdx.x);
  if (it.seg < 0) return;
  const size_t unit = static_cast<size_t>(blockIdx.x) * a.heads + h;
  const int n = it.count, kc = dim / 8, r_step = 128 / kc, c_step = 128 % kc;
  for (int r = static_cast<int>(threadIdx.x) / kc, c = static_cast<int>(threadIdx.x) % kc; r < kChunk;) {
    uint4 q = make_uint4(0u, 0u, 0u, 0u), k = q;
    if (r < n) {
      const size_t off = static_cast<size_t>(it.row0 + r) * a.stride + static_cast<size_t>(kh) * dim + c * 8;
      q = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.q) + off);
      k = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.k) + off);
    }
    *reinterpret_cast<uint4*>(s_q + r * pitch + c * 8) = q;
    *reinterpret_cast<uint4*>(s_k + r * pitch + c * 8) = k;
    r += r_step;
    c += c_step;
    if (c >= kc) { c -= kc; ++r; }
  }
  for (int i = threadIdx.x; i < kChunk * kPitch; i += 128) s_m[i] = 0.f;
  if (warp == 0) {                     // gates and the running sum of log decays
    float last = 0.f;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int r = u * 32 + lane;
      float beta = 0.f, c = 0.f;
      if (r < n) delta_gates(a, static_cast<size_t>(it.row0) + r, h, &beta, &c);
#pragma unroll
      for (int off = 1; off < 32; off <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, c, off);
        if (lane >= off) c += up;
      }
      c += last;
      last = __shfl_sync(0xffffffffu, c, 31);
      s_row[r].x = c;
      s_row[r].y = beta;
    }
  }
  __syncthreads();
  {                                    // lengths: two threads per row
    const int r = threadIdx.x >> 1, half = threadIdx.x & 1;
    float kk = 0.f, qq = 0.f;
    for (int c = half; c < kc; c += 2) {
      float x[8];
      VecIO<__nv_bfloat16, 8>::ld(s_k + r * pitch + c * 8, x);
#pragma unroll
      for (int i = 0; i < 8; ++i) kk = fmaf(x[i], x[i], kk);
      VecIO<__nv_bfloat16, 8>::ld(s_q + r * pitch + c * 8, x);
#pragma unroll
      for (int i = 0; i < 8; ++i) qq = fmaf(x[i], x[i], qq);
    }
    kk += __shfl_xor_sync(0xffffffffu, kk, 1);
    qq += __shfl_xor_sync(0xffffffffu, qq, 1);
    if (half == 0) {
      s_row[r].z = 1.f / sqrtf(kk + kUnitEps);
      s_row[r].w = 1.f / (sqrtf(qq + kUnitEps) * sqrtf(static_cast<float>(dim)));
    }
  }
  __syncthreads();
  if (threadIdx.x < kChunk) ws.rows[unit * kChunk + threadIdx.x] = s_row[threadIdx.x];
  // K K^T and Q K^T up to the diagonal
  float kk[8][4], qk[8][4];
#pragma unroll
  for (int nn = 0; nn < 8; ++nn)
#pragma unroll
    for (int e = 0; e < 4; ++e) kk[nn][e] = qk[nn][e] = 0.f;
  const uint32_t row_off = ((warp * 16 + (lane & 15)) * pitch + (lane >> 4) * 8) * 2;
  const uint32_t ka = smem_addr(s_k) + (((lane & 7) + ((lane >> 4) << 3)) * pitch + ((lane >> 3) & 1) * 8) * 2;
  for (int k = 0; k < dim / 16; ++k) {
    uint32_t fk[4], fq[4];
    ldsm_x4(smem_addr(s_k) + row_off + k * 32, fk);
    ldsm_x4(smem_addr(s_q) + row_off + k * 32, fq);
#pragma unroll
    for (int nn = 0; nn < 8; nn += 2) {
      if (nn <= 2 * warp + 1) {
        uint32_t b[4];
        ldsm_x4(ka + nn * 8 * pitch * 2 + k * 32, b);
        mma_bf16(kk[nn], fk, b[0], b[1]);
        mma_bf16(kk[nn + 1], fk, b[2], b[3]);
        mma_bf16(qk[nn], fq, b[0], b[1]);
        mma_bf16(qk[nn + 1], fq, b[2], b[3]);
      }
    }
  }
  const int i0 = warp * 16 + (lane >> 2);
#pragma unroll
  for (int kt = 0; kt < 4; ++kt) {
    if (kt > warp) continue;
    float p[2][4];
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = i0 + (e >> 1) * 8, j = kt * 16 + u * 8 + (lane & 3) * 2 + (e & 1);
        const float4 ri = s_row[i], rj = s_row[j];
        const float d = j <= i ? __expf(ri.x - rj.x) * rj.z : 0.f;
        p[u][e] = qk[2 * kt + u][e] * d * ri.w;
        s_a[i * kPitch + j] = j < i ? kk[2 * kt + u][e] * d * ri.z * ri.y : 0.f;
      }
    uint4 hi, lo;
    split_pair(p[0][0], p[0][1], &hi.x, &lo.x);
    split_pair(p[0][2], p[0][3], &hi.y, &lo.y);
    split_pair(p[1][0], p[1][1], &hi.z, &lo.z);
    split_pair(p[1][2], p[1][3], &hi.w, &lo.w);
    uint4* dst = tile_at(ws, unit, 1, warp, kt);
    dst[lane] = hi;
    dst[32 + lane] = lo;
  }
  __syncwarp();
  // (I + A)^-1: diagonal blocks column by column, a warp each (its own rows of A are its own writes)
  {
    const int b = warp * 16;
    if (lane < 16) {
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float t = i == lane ? 1.f : 0.f;
#pragma unroll
        for (int j = 0; j < 16; ++j)
          if (j < i) t = fmaf(-s_a[(b + i) * kPitch + b + j], x[j], t);
        x[i] = t;
      }
#pragma unroll
      for (int i = 0; i < 16; ++i) s_m[(b + i) * kPitch + b + lane] = x[i];
    }
  }
  __syncthreads();
  // lower left blocks of size m from the diagonal ones: -M22 (A21 M11); a thread has ROWS rows of four columns
  auto lower_left = [&](auto size, auto count) {
    constexpr int m = decltype(size)::value, ROWS = decltype(count)::value, kPitchT = 36;
    const int unit_rows = m / ROWS, units = unit_rows * (m / 4), pair = static_cast<int>(threadIdx.x) / units, at = static_cast<int>(threadIdx.x) % units;
    const int r0 = at / (m / 4) * ROWS, c0 = at % (m / 4) * 4, b = pair * 2 * m;
    float* t = s_t + pair * m * kPitchT;
    auto product = [&](const float* x, const float* y, int y_pitch, int from, int to, float (&out)[ROWS][4]) {
#pragma unroll
      for (int r = 0; r < ROWS; ++r)
#pragma unroll
        for (int e = 0; e < 4; ++e) out[r][e] = 0.f;
      for (int j = from; j < to; ++j) {
        const float4 v = *reinterpret_cast<const float4*>(y + j * y_pitch);
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
          const float f = x[r * kPitch + j];
          out[r][0] = fmaf(f, v.x, out[r][0]); out[r][1] = fmaf(f, v.y, out[r][1]); out[r][2] = fmaf(f, v.z, out[r][2]); out[r][3] = fmaf(f, v.w, out[r][3]);
        }
      }
    };
    float out[ROWS][4];
    product(s_a + (b + m + r0) * kPitch + b, s_m + b * kPitch + b + c0, kPitch, c0, m, out);
#pragma unroll
    for (int r = 0; r < ROWS; ++r) *reinterpret_cast<float4*>(t + (r0 + r) * kPitchT + c0) = make_float4(out[r][0], out[r][1], out[r][2], out[r][3]);
    __syncthreads();
    product(s_m + (b + m + r0) * kPitch + b + m, t + c0, kPitchT, 0, r0 + ROWS, out);
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
      *reinterpret_cast<float4*>(s_m + (b + m + r0 + r) * kPitch + b + c0) = make_float4(-out[r][0], -out[r][1], -out[r][2], -out[r][3]);
    __syncthreads();
  };
  lower_left(std::integral_constant<int, 16>{}, std::integral_constant<int, 1>{});
  lower_left(std::integral_constant<int, 32>{}, std::integral_constant<int, 2>{});
#pragma unroll
  for (int kt = 0; kt < 4; ++kt) {
    if (kt > warp) continue;
    const float* m0 = s_m + i0 * kPitch + kt * 16 + (lane & 3) * 2;
    auto entry = [&](int dr, int dc) { return m0[dr * kPitch + dc]; };
    uint4 hi, lo;
    split_pair(entry(0, 0), entry(0, 1), &hi.x, &lo.x);
    split_pair(entry(8, 0), entry(8, 1), &hi.y, &lo.y);
    split_pair(entry(0, 8), entry(0, 9), &hi.z, &lo.z);
    split_pair(entry(8, 8), entry(8, 9), &hi.w, &lo.w);
    uint4* dst = tile_at(ws, unit, 0, warp, kt);
    dst[lane] = hi;
    dst[32 + lane] = lo;
  }
}

// Warps 0..3 have the keys' side (16 tokens each: K S, the right-hand sides, the writes U), warps 4..7 the queries' (Q S, P U, the
// output); all eight have a 16-row tile of the state. NT 8-column tiles of the values per CTA.
constexpr int kChainThreads = 256;
template <int NT>
__global__ void __launch_bounds__(kChainThreads)
delta_chain_kernel(const Args a, const ChunkSpace ws) {
  constexpr int kCols = NT * 8, kPitchC = kCols + 8;
  extern __shared__ __align__(16) uint8_t raw[];
  const int dim = a.dim, pitch = dim + 8;
  __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(raw);        // [2][64][pitch]
  __nv_bfloat16* s_k = s_q + 2 * kChunk * pitch;                     // [2][64][pitch]
  __nv_bfloat16* s_s = s_k + 2 * kChunk * pitch;                     // [hi, lo][dim][kPitchC] state
  __nv_bfloat16* s_r = s_s + 2 * dim * kPitchC;                      // [hi, lo][64][kPitchC] right-hand sides
  __nv_bfloat16* s_u = s_r + 2 * kChunk * kPitchC;                   // [hi, lo][64][kPitchC] writes
  __nv_bfloat16* s_d = s_u + 2 * kChunk * kPitchC;                   // [hi, lo][64][kPitchC] writes, decayed to the chunk's end
  float4* s_row = reinterpret_cast<float4*>(s_d + 2 * kChunk * kPitchC);      // [2][64]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, band = warp & 3;
  const bool keys = warp < 4;
  const int seg = blockIdx.x, h = blockIdx.y, kh = key_head(a, h), v0 = blockIdx.z * kCols;
  const int row0 = a.cu_rows[seg], rows = a.cu_rows[seg + 1] - row0;
  if (rows <= 0) return;
  int first = 0;
  for (int s = 0; s < seg; ++s) first += (a.cu_rows[s + 1] - a.cu_rows[s] + kChunk - 1) / kChunk;
  const int chunks = (rows + kChunk - 1) / kChunk, cols = min(kCols, a.vdim - v0), kc = dim / 8;

  const int r_first = static_cast<int>(threadIdx.x) / kc, c_first = static_cast<int>(threadIdx.x) % kc, r_step = kChainThreads / kc, c_step = kChainThreads % kc;
  auto fetch = [&](int chunk) {        // q, k and the rows' numbers of a chunk, asynchronously
    const int buf = chunk & 1, n = min(kChunk, rows - chunk * kChunk);
    for (int r = r_first, c = c_first; r < kChunk;) {
      const size_t off = static_cast<size_t>(row0 + chunk * kChunk + min(r, n - 1)) * a.stride + static_cast<size_t>(kh) * dim + c * 8;
      const int bytes = r < n ? 16 : 0;      // (rows behind the last are zero)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(s_q + (buf * kChunk + r) * pitch + c * 8)),
                   "l"(static_cast<const __nv_bfloat16*>(a.q) + off), "r"(bytes) : "memory");
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(s_k + (buf * kChunk + r) * pitch + c * 8)),
                   "l"(static_cast<const __nv_bfloat16*>(a.k) + off), "r"(bytes) : "memory");
      r += r_step;
      c += c_step;
      if (c >= kc) { c -= kc; ++r; }
    }
    if (threadIdx.x < kChunk) {
      const float4* src = ws.rows + (static_cast<size_t>(first + chunk) * a.heads + h) * kChunk + threadIdx.x;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(s_row + buf * kChunk + threadIdx.x)), "l"(src) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);

  float* state = slot_state(a, seg, h) + v0;
  const bool fresh = a.positions[row0] == 0;
  const int m0 = warp * 16;            // this warp's rows of the state
  float st[NT][4];
#pragma unroll
  for (int nn = 0; nn < NT; ++nn)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int d = m0 + (lane >> 2) + e * 8, c = nn * 8 + (lane & 3) * 2;
      float2 x = make_float2(0.f, 0.f);
      if (!fresh && d < dim && c < cols) x = *reinterpret_cast<const float2*>(state + static_cast<size_t>(d) * a.vdim + c);
      st[nn][e * 2] = x.x;
      st[nn][e * 2 + 1] = x.y;
    }

  const int i0 = band * 16 + (lane >> 2);
  const uint32_t frag_row = ((band * 16 + (lane & 15)) * pitch + (lane >> 4) * 8) * 2;
  const uint32_t frag_b = (((lane & 7) + ((lane >> 3) & 1) * 8) * kPitchC + (lane >> 4) * 8) * 2;
  const uint32_t frag_kt = (((lane & 7) + ((lane >> 4) & 1) * 8) * pitch + ((lane >> 3) & 1) * 8) * 2;
  // C fragments of rows i0, i0 + 8 as two bf16 planes
  auto leave = [&](__nv_bfloat16* dst, const float (&x)[NT][4], float f0, float f1) {
#pragma unroll
    for (int nn = 0; nn < NT; ++nn)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float f = e ? f1 : f0;
        uint32_t hi, lo;
        split_pair(x[nn][e * 2] * f, x[nn][e * 2 + 1] * f, &hi, &lo);
        const int at = (i0 + e * 8) * kPitchC + nn * 8 + (lane & 3) * 2;
        *reinterpret_cast<uint32_t*>(dst + at) = hi;
        *reinterpret_cast<uint32_t*>(dst + kChunk * kPitchC + at) = lo;
      }
  };
  // y += (hi + lo)[64 rows of a triangle's row tile] x [64][columns], the product of the two small parts left out
  uint4 hi[4], lo[4];                  // this warp's row tile of M (keys) or P (queries)
  auto triangle = [&](const __nv_bfloat16* x, float (&y)[NT][4]) {
    const uint32_t xb = smem_addr(x) + frag_b;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      if (kt > band) continue;
      const uint32_t ah[4] = {hi[kt].x, hi[kt].y, hi[kt].z, hi[kt].w}, al[4] = {lo[kt].x, lo[kt].y, lo[kt].z, lo[kt].w};
#pragma unroll
      for (int nn = 0; nn < NT; nn += 2) {
        uint32_t b[4], bl[4];
        ldsm_x4_t(xb + (kt * 16 * kPitchC + nn * 8) * 2, b);
        ldsm_x4_t(xb + ((kChunk + kt * 16) * kPitchC + nn * 8) * 2, bl);
        mma_bf16(y[nn], ah, b[0], b[1]);
        mma_bf16(y[nn + 1], ah, b[2], b[3]);
        mma_bf16(y[nn], al, b[0], b[1]);
        mma_bf16(y[nn + 1], al, b[2], b[3]);
        mma_bf16(y[nn], ah, bl[0], bl[1]);
        mma_bf16(y[nn + 1], ah, bl[2], bl[3]);
      }
    }
  };

  for (int chunk = 0; chunk < chunks; ++chunk) {
    const int buf = chunk & 1, n = min(kChunk, rows - chunk * kChunk);
    const size_t unit = static_cast<size_t>(first + chunk) * a.heads + h;
    const size_t base = static_cast<size_t>(row0) + chunk * kChunk;
    // operands of this chunk that wait for nothing
#pragma unroll
    for (int kt = 0; kt < 4; ++kt)
      if (kt <= band) {
        const uint4* m = tile_at(ws, unit, keys ? 0 : 1, band, kt);
        hi[kt] = m[lane];
        lo[kt] = m[32 + lane];
      }
    uint32_t v[NT][2];
#pragma unroll
    for (int nn = 0; nn < NT; ++nn)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = i0 + e * 8, c = nn * 8 + (lane & 3) * 2;
        v[nn][e] = keys && r < n && c < cols ? *reinterpret_cast<const uint32_t*>(static_cast<const __nv_bfloat16*>(a.v) + (base + r) * a.stride +
                                                                                 static_cast<size_t>(h) * a.vdim + v0 + c) : 0u;
      }
#pragma unroll
    for (int nn = 0; nn < NT; ++nn)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = m0 + (lane >> 2) + e * 8, c = nn * 8 + (lane & 3) * 2;
        if (d < dim) {
          uint32_t sh, sl;
          split_pair(st[nn][e * 2], st[nn][e * 2 + 1], &sh, &sl);
          *reinterpret_cast<uint32_t*>(s_s + d * kPitchC + c) = sh;
          *reinterpret_cast<uint32_t*>(s_s + (dim + d) * kPitchC + c) = sl;
        }
      }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                   // this chunk's rows and state are there, the other buffer and the writes are free
    if (chunk + 1 < chunks) fetch(chunk + 1);

    float x[2][NT][4];                 // K S or Q S, the state's two parts in sums of their own
#pragma unroll
    for (int part = 0; part < 2; ++part)
#pragma unroll
      for (int nn = 0; nn < NT; ++nn)
#pragma unroll
        for (int e = 0; e < 4; ++e) x[part][nn][e] = 0.f;
    const uint32_t ka = smem_addr(s_k + buf * kChunk * pitch), own = (keys ? ka : smem_addr(s_q + buf * kChunk * pitch)) + frag_row;
    const uint32_t sb = smem_addr(s_s) + frag_b;
#pragma unroll 4
    for (int k = 0; k < dim / 16; ++k) {
      uint32_t f[4];
      ldsm_x4(own + k * 32, f);
#pragma unroll
      for (int part = 0; part < 2; ++part)
#pragma unroll
        for (int nn = 0; nn < NT; nn += 2) {
          uint32_t b[4];
          ldsm_x4_t(sb + ((part * dim + k * 16) * kPitchC + nn * 8) * 2, b);
          mma_bf16(x[part][nn], f, b[0], b[1]);
          mma_bf16(x[part][nn + 1], f, b[2], b[3]);
        }
    }
    const float4 ra = s_row[buf * kChunk + i0], rb = s_row[buf * kChunk + i0 + 8];      // (c, beta, 1/|k|, 1/|q|)
    const float end = s_row[buf * kChunk + kChunk - 1].x;
    const float ea = __expf(ra.x) * (keys ? ra.z : ra.w), eb = __expf(rb.x) * (keys ? rb.z : rb.w);
    float y[NT][4];
    if (keys) {
#pragma unroll
      for (int nn = 0; nn < NT; ++nn) {
        y[nn][0] = ra.y * (__uint_as_float(v[nn][0] << 16) - ea * (x[0][nn][0] + x[1][nn][0]));
        y[nn][1] = ra.y * (__uint_as_float(v[nn][0] & 0xffff0000u) - ea * (x[0][nn][1] + x[1][nn][1]));
        y[nn][2] = rb.y * (__uint_as_float(v[nn][1] << 16) - eb * (x[0][nn][2] + x[1][nn][2]));
        y[nn][3] = rb.y * (__uint_as_float(v[nn][1] & 0xffff0000u) - eb * (x[0][nn][3] + x[1][nn][3]));
      }
      leave(s_r, y, 1.f, 1.f);
      asm volatile("barrier.cta.sync 1, 128;" ::: "memory");
#pragma unroll
      for (int nn = 0; nn < NT; ++nn)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[nn][e] = 0.f;
      triangle(s_r, y);
      leave(s_u, y, 1.f, 1.f);
      leave(s_d, y, __expf(end - ra.x) * ra.z, __expf(end - rb.x) * rb.z);
    } else {
#pragma unroll
      for (int nn = 0; nn < NT; ++nn) {
        y[nn][0] = ea * (x[0][nn][0] + x[1][nn][0]); y[nn][1] = ea * (x[0][nn][1] + x[1][nn][1]);
        y[nn][2] = eb * (x[0][nn][2] + x[1][nn][2]); y[nn][3] = eb * (x[0][nn][3] + x[1][nn][3]);
      }
    }
    __syncthreads();                   // the writes are there
    const float keep = __expf(end);
    if (m0 < dim) {
      const uint32_t db = smem_addr(s_d) + frag_b;
#pragma unroll
      for (int nn = 0; nn < NT; ++nn)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[nn][e] *= keep;
#pragma unroll
      for (int k = 0; k < kChunk / 16; ++k) {
        uint32_t af[4];
        ldsm_x4_t(ka + frag_kt + (k * 16 * pitch + m0) * 2, af);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int nn = 0; nn < NT; nn += 2) {
            uint32_t b[4];
            ldsm_x4_t(db + ((part * kChunk + k * 16) * kPitchC + nn * 8) * 2, b);
            mma_bf16(st[nn], af, b[0], b[1]);
            mma_bf16(st[nn + 1], af, b[2], b[3]);
          }
      }
    }
    if (!keys) {
      triangle(s_u, y);
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = i0 + e * 8;
        if (i < n) {
          __nv_bfloat16* dst = out + ((base + i) * a.heads + h) * a.vdim + v0;
#pragma unroll
          for (int nn = 0; nn < NT; ++nn) {
            const int c = nn * 8 + (lane & 3) * 2;
            if (c < cols) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(y[nn][e * 2], y[nn][e * 2 + 1]);
          }
        }
      }
    }
  }
#pragma unroll
  for (int nn = 0; nn < NT; ++nn)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int d = m0 + (lane >> 2) + e * 8, c = nn * 8 + (lane & 3) * 2;
      if (d < dim && c < cols) *reinterpret_cast<float2*>(state + static_cast<size_t>(d) * a.vdim + c) = make_float2(st[nn][e * 2], st[nn][e * 2 + 1]);
    }
}

bool delta_args_ok(const Args& a) {
  return a.positions && a.cu_rows && a.slots && a.q && a.k && a.v && a.z && a.bias && a.log_rate && a.state && a.out && a.segments > 0 && a.heads > 0 &&
         a.heads <= 65535 && a.key_heads > 0 && a.heads % a.key_heads == 0 && a.dim > 0 && a.vdim > 0 && a.num_slots > 0 && a.z_stride >= 2ll * a.heads &&
         a.slot_stride >= static_cast<long long>(a.heads) * a.dim * a.vdim;
}

template <typename T>
int launch_simple(const Args& a, cudaStream_t st) {
  const size_t smem = (static_cast<size_t>(a.dim) * 34 + 512 + 32) * 4;
  if (smem > 200 * 1024) return CACHEIR_B200_ELIMIT;
  const cudaError_t e = cudaFuncSetAttribute(delta_simple_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  delta_simple_kernel<T><<<dim3(a.segments, a.heads, (a.vdim + 31) / 32), 256, smem, st>>>(a);
  return launch_status();
}

template <typename T>
int launch_step(const Args& a, const void* gate, long long gate_stride, const float* w, float eps, cudaStream_t st) {
  const dim3 grid(a.segments, a.heads);
  const size_t smem = static_cast<size_t>(a.dim) * 8;
  const int per_row = a.vdim / 4;
#define CB200_DELTA_STEP(THREADS, HELD) \
  delta_step_kernel<T, THREADS, HELD><<<grid, THREADS, smem, st>>>(a, static_cast<const T*>(gate), gate_stride, w, eps)
  if (a.dim <= 256 / per_row * 4) CB200_DELTA_STEP(256, 4);
  else if (a.dim <= 256 / per_row * 16) CB200_DELTA_STEP(256, 16);
  else CB200_DELTA_STEP(512, 16);
#undef CB200_DELTA_STEP
  return launch_status();
}

template <int NT>
int launch_chain(const Args& a, const ChunkSpace& ws, cudaStream_t st) {
  constexpr int kCols = NT * 8, kPitchC = kCols + 8;
  auto kern = delta_chain_kernel<NT>;
  const size_t smem = (static_cast<size_t>(4) * kChunk * (a.dim + 8) + static_cast<size_t>(2) * (a.dim + 3 * kChunk) * kPitchC) * 2 + 2 * kChunk * 16;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(a.segments, a.heads, (a.vdim + kCols - 1) / kCols), kChainThreads, smem, st>>>(a, ws);
  return launch_status();
}

size_t unit_bytes() { return static_cast<size_t>(2) * kTri * 64 * 16 + kChunk * 16; }

}  // namespace
}  // namespace cb200

using namespace cb200;

extern "C" int cacheir_b200_delta_simple(const cacheir_b200_delta_args* a, void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (!delta_args_ok(*a)) return CACHEIR_B200_EINVAL;
  CB200_HYBRID_DTYPE(a->dtype, return launch_simple<T>(*a, as_stream(stream)));
  return CACHEIR_B200_EUNSUPPORTED;
}

extern "C" int cacheir_b200_delta_step(const cacheir_b200_delta_args* a, const void* gate, long long gate_stride, const float* w, float eps,
                                       void* stream) {
  if (!a) return CACHEIR_B200_EINVAL;
  if (a->rows <= 0) return 0;
  if (!delta_args_ok(*a) || !gate || !w || a->rows != a->segments) return CACHEIR_B200_EINVAL;
  if (a->vdim % 4 != 0 || a->vdim > 1024 || a->dim > 4096) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(a->state, 16) || a->slot_stride % 4 != 0) return CACHEIR_B200_EALIGN;
  CB200_HYBRID_DTYPE(a->dtype, return launch_step<T>(*a, gate, gate_stride, w, eps, as_stream(stream)));
  return CACHEIR_B200_EUNSUPPORTED;
}

extern "C" int cacheir_b200_delta_chunked_supported(int dim, int vdim, int dtype) {
  return dtype == CACHEIR_B200_BF16 && dim >= 16 && dim % 16 == 0 && dim <= 128 && vdim % 8 == 0 ? 1 : 0;
}

extern "C" size_t cacheir_b200_delta_workspace_bytes(int rows, int segments, int heads) {
  return static_cast<size_t>(ragged_items(rows, segments, kChunk)) * heads * unit_bytes();
}

extern "C" int cacheir_b200_delta_chunked(const cacheir_b200_delta_args* args, void* workspace, size_t workspace_bytes, void* stream) {
  if (!args) return CACHEIR_B200_EINVAL;
  const cacheir_b200_delta_args& a = *args;
  if (a.rows <= 0) return 0;
  if (!delta_args_ok(a)) return CACHEIR_B200_EINVAL;
  if (!cacheir_b200_delta_chunked_supported(a.dim, a.vdim, a.dtype)) return CACHEIR_B200_EUNSUPPORTED;
  if (!aligned_to(a.q, 16) || !aligned_to(a.k, 16) || !aligned_to(a.v, 16) || !aligned_to(a.out, 16) || a.stride % 8 != 0 ||
      !aligned_to(a.state, 16) || a.slot_stride % 4 != 0 || !aligned_to(workspace, 16))
    return CACHEIR_B200_EALIGN;
  if (!workspace || workspace_bytes < cacheir_b200_delta_workspace_bytes(a.rows, a.segments, a.heads)) return CACHEIR_B200_EWORKSPACE;
  const int items = ragged_items(a.rows, a.segments, kChunk);
  const size_t units = static_cast<size_t>(items) * a.heads;
  ChunkSpace ws;
  ws.tiles = static_cast<uint4*>(workspace);
  ws.rows = reinterpret_cast<float4*>(ws.tiles + units * 2 * kTri * 64);
  cudaStream_t st = as_stream(stream);
  const size_t smem = static_cast<size_t>(2) * kChunk * (a.dim + 8) * 2 + (static_cast<size_t>(2) * kChunk * (kChunk + 4) + 32 * 36) * 4;
  const cudaError_t e = cudaFuncSetAttribute(delta_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  delta_local_kernel<<<dim3(items, a.heads), 128, smem, st>>>(a, ws);
  const int rc = launch_status();
  if (rc != 0) return rc;
  // narrow column blocks while all of them still run at once
  const bool narrow = static_cast<long long>(a.segments) * a.heads * ((a.vdim + 15) / 16) <= kNumSMs;
  return narrow ? launch_chain<2>(a, ws, st) : launch_chain<4>(a, ws, st);
}

extern "C" int cacheir_b200_delta_device_status(int) { return 0; }
