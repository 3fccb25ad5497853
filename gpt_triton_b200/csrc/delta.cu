// Gated delta rule.  Per head with an fp32 state S [dim, vdim], one decay g and one step size beta per token:
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// q, k, v pass a short causal convolution per channel and silu; q and k become unit vectors.
//
// One token:
//   delta_token_kernel     everything in one kernel, the state through shared memory (heads up to 256 columns each)
// A few tokens, or fp32 (heads up to 128 x 256):
//   delta_step_kernel      everything in one kernel, token by token; the state of a head in the registers of one block
// Many tokens, bf16 (delta_chunk.cu): 64 tokens at a time on the tensor cores.
// Any other size:
//   delta_inputs_kernel    convolution and silu (stored in the operand type), 1 / |q|, 1 / |k| of what is stored, log decays and
//                          step sizes in fp32
//   delta_any_kernel       the recurrence token by token, state in global memory
// conv_store_kernel puts the last inputs of the convolutions into the ring that remembers them.
#include <atomic>

#include "common.cuh"

namespace b200 {
namespace {

__device__ __forceinline__ float silu_exact(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_exact(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

// ------------------------------------------------------------------ convolution, unit norms, gates
constexpr int kInputWarps = 8, kInputTokens = 16;

// One input of the convolution at position `pos` of sequence b: a row of this call, the ring's memory, or zero.
template <typename T>
__device__ __forceinline__ float conv_input(const b200_delta_args& p, int64_t b, int64_t t, int64_t pos, int64_t c) {
  if (t >= 0) return to_float(static_cast<const T*>(p.rows)[(b * p.n + t) * p.ld + c]);
  if (pos < 0) return 0.f;
  return to_float(static_cast<const T*>(p.conv_state)[(b * p.taps + pos % p.taps) * p.conv_cols + c]);
}

template <typename T>
__global__ void __launch_bounds__(32 * kInputWarps)
delta_inputs_kernel(b200_delta_args p, int64_t tiles) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t b = blockIdx.x / tiles, t0 = (blockIdx.x % tiles) * kInputTokens;
  const int64_t start = p.pos_dev ? (int64_t)p.pos_dev[0] : p.start;
  const int nt = (int)(p.n - t0 < kInputTokens ? p.n - t0 : kInputTokens);
  const int64_t M = p.B * p.n;
  const int taps = (int)p.taps;
  const int sections = (int)(2 * p.kv_heads + p.heads);
  for (int s = warp; s < sections; s += kInputWarps) {
    const bool is_v = s >= 2 * p.kv_heads, is_k = !is_v && s >= p.kv_heads;
    const int width = (int)(is_v ? p.vdim : p.dim);
    const int64_t c0 = is_v ? p.off_v + (s - 2 * p.kv_heads) * p.vdim : is_k ? p.off_k + (s - p.kv_heads) * p.dim : s * p.dim;
    for (int i = 0; i < nt; ++i) {
      const int64_t t = t0 + i, row = b * p.n + t;
      float sq = 0.f;
      for (int c = lane; c < width; c += 32) {
        float a = 0.f;
        for (int k = 0; k < taps; ++k) {
          const int64_t back = taps - 1 - k;
          a = fmaf(p.conv_w[(c0 + c) * taps + k], conv_input<T>(p, b, t - back, start + t - back, c0 + c), a);
        }
        const T o = from_float<T>(silu_exact(a));
        static_cast<T*>(p.mixed)[row * p.ld_mixed + c0 + c] = o;
        const float f = to_float(o);
        sq = fmaf(f, f, sq);
      }
      if (!is_v) {
        sq = warp_sum(sq);
        if (lane == 0) p.norms[(int64_t)s * M + row] = (is_k ? 1.0f : p.q_scale) / sqrtf(sq + p.unit_eps);
      }
    }
  }
  for (int64_t i = threadIdx.x; i < nt * p.heads; i += 32 * kInputWarps) {
    const int64_t h = i / nt, row = b * p.n + t0 + i % nt;
    const T* src = static_cast<const T*>(p.rows) + row * p.ld;
    p.gates[h * M + row] = -expf(p.a_log[h]) * softplus_exact(to_float(src[p.off_a + h]) + p.dt_bias[h]);
    p.gates[(p.heads + h) * M + row] = 1.0f / (1.0f + expf(-to_float(src[p.off_b + h])));
  }
}

// Positions [end - (taps - 1), end) of this call's inputs into slot position % taps (a slot is read for at most taps - 1
// positions, so the oldest one may be overwritten by the newest).
template <typename T>
__global__ void __launch_bounds__(256)
conv_store_kernel(b200_delta_args p) {
  const int64_t b = blockIdx.x;
  const int64_t start = p.pos_dev ? (int64_t)p.pos_dev[0] : p.start;
  const int64_t first = p.n > p.taps - 1 ? p.n - (p.taps - 1) : 0;
  for (int64_t t = first; t < p.n; ++t) {
    const T* src = static_cast<const T*>(p.rows) + (b * p.n + t) * p.ld;
    T* dst = static_cast<T*>(p.conv_state) + (b * p.taps + (start + t) % p.taps) * p.conv_cols;
    for (int64_t c = (int64_t)blockIdx.y * 256 + threadIdx.x; c < p.conv_cols; c += (int64_t)gridDim.y * 256) dst[c] = src[c];
  }
}

// ------------------------------------------------------------------ token by token, any sizes
constexpr int kAnyThreads = 128;
template <typename T>
__global__ void __launch_bounds__(kAnyThreads)
delta_any_kernel(b200_delta_args p) {
  extern __shared__ float smem_f[];
  __shared__ float part[kAnyThreads / 32];
  const int dim = (int)p.dim, vdim = (int)p.vdim;
  float *qs = smem_f, *ks = qs + dim, *os = ks + dim;
  const int64_t h = blockIdx.x % p.heads, b = blockIdx.x / p.heads, kv = h / (p.heads / p.kv_heads), M = p.B * p.n;
  float* S = p.state + (b * p.heads + h) * (int64_t)dim * vdim;
  const T* mixed = static_cast<const T*>(p.mixed);
  for (int64_t t = 0; t < p.n; ++t) {
    const int64_t row = b * p.n + t;
    const T* src = mixed + row * p.ld_mixed;
    const float rq = p.norms[kv * M + row], rk = p.norms[(p.kv_heads + kv) * M + row];
    const float g = expf(p.gates[h * M + row]), beta = p.gates[(p.heads + h) * M + row];
    for (int i = threadIdx.x; i < dim; i += kAnyThreads) qs[i] = to_float(src[kv * dim + i]) * rq, ks[i] = to_float(src[p.off_k + kv * dim + i]) * rk;
    __syncthreads();
    const bool zero = p.fresh && t == 0;
    float sq = 0.f;
    for (int c = threadIdx.x; c < vdim; c += kAnyThreads) {
      float seen = 0.f;
      if (!zero)
        for (int i = 0; i < dim; ++i) seen = fmaf(S[(int64_t)i * vdim + c] * g, ks[i], seen);
      const float u = beta * (to_float(src[p.off_v + h * vdim + c]) - seen);
      float o = 0.f;
      for (int i = 0; i < dim; ++i) {
        const float s = fmaf(ks[i], u, zero ? 0.f : S[(int64_t)i * vdim + c] * g);
        S[(int64_t)i * vdim + c] = s;
        o = fmaf(s, qs[i], o);
      }
      os[c] = o;
      sq = fmaf(o, o, sq);
    }
    sq = warp_sum(sq);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = sq;
    __syncthreads();
    sq = 0.f;
    for (int i = 0; i < kAnyThreads / 32; ++i) sq += part[i];
    const float inv = 1.0f / sqrtf(sq / (float)vdim + p.eps);
    const T* gate = static_cast<const T*>(p.rows) + row * p.ld + p.off_g + h * vdim;
    T* y = static_cast<T*>(p.y) + row * p.ld_y + h * vdim;
    for (int c = threadIdx.x; c < vdim; c += kAnyThreads) y[c] = from_float<T>(os[c] * inv * p.norm_w[c] * to_float(gate[c]));
    __syncthreads();
  }
}

// ------------------------------------------------------------------ token by token, the state in registers
// One block per (sequence, head): four row groups of warps (ROWS = 16 or 32 state rows each) x one group per 32 columns.
constexpr int kStepRowWarps = 4, kStepMaxCols = 256;

template <typename T, int ROWS, int THREADS>
__global__ void __launch_bounds__(THREADS, 1)
delta_step_kernel(b200_delta_args p) {
  constexpr int DIM = kStepRowWarps * ROWS;
  __shared__ __align__(16) float qs[DIM], ks[DIM];
  __shared__ float vs[kStepMaxCols], part[kStepRowWarps][kStepMaxCols], red[3][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const int rw = warp % kStepRowWarps, col = (warp / kStepRowWarps) * 32 + lane, row0 = rw * ROWS;
  const int dim = (int)p.dim, vdim = (int)p.vdim, taps = (int)p.taps;
  const int64_t h = blockIdx.x % p.heads, b = blockIdx.x / p.heads, group = p.heads / p.kv_heads, kv = h / group;
  const int64_t start = p.pos_dev ? (int64_t)p.pos_dev[0] : p.start;
  const bool col_ok = col < vdim;
  float* st = p.state + (b * p.heads + h) * (int64_t)dim * vdim + col;
  float s[ROWS];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) s[i] = (!p.fresh && col_ok && row0 + i < dim) ? st[(int64_t)(row0 + i) * vdim] : 0.f;
  const float decay_rate = -expf(p.a_log[h]), dt_bias = p.dt_bias[h];
  const int channels = 2 * dim + vdim;
  for (int64_t t = 0; t < p.n; ++t) {
    const int64_t row = b * p.n + t;
    const T* src = static_cast<const T*>(p.rows) + row * p.ld;
    // convolutions and silu: q, then k, then v channels
    float sq_q = 0.f, sq_k = 0.f;
    for (int c = threadIdx.x; c < channels; c += blockDim.x) {
      const int64_t col_in = c < dim ? kv * dim + c : c < 2 * dim ? p.off_k + kv * dim + (c - dim) : p.off_v + h * vdim + (c - 2 * dim);
      float a = 0.f;
      for (int k = 0; k < taps; ++k) {
        const int64_t back = taps - 1 - k;
        a = fmaf(p.conv_w[col_in * taps + k], conv_input<T>(p, b, t - back, start + t - back, col_in), a);
      }
      const float o = to_float(from_float<T>(silu_exact(a)));
      if (c < dim) qs[c] = o, sq_q = fmaf(o, o, sq_q);
      else if (c < 2 * dim) ks[c - dim] = o, sq_k = fmaf(o, o, sq_k);
      else vs[c - 2 * dim] = o;
    }
    // (rows of the state beyond dim see a key and a query of zero)
    for (int c = dim + threadIdx.x; c < DIM; c += blockDim.x) qs[c] = 0.f, ks[c] = 0.f;
    sq_q = warp_sum(sq_q), sq_k = warp_sum(sq_k);
    if (lane == 0) red[0][warp] = sq_q, red[1][warp] = sq_k;
    const float g = expf(decay_rate * softplus_exact(to_float(src[p.off_a + h]) + dt_bias));
    const float beta = 1.0f / (1.0f + expf(-to_float(src[p.off_b + h])));
    __syncthreads();
    float rq = 0.f, rk = 0.f;
    for (int i = 0; i < n_warps; ++i) rq += red[0][i], rk += red[1][i];
    rq = p.q_scale / sqrtf(rq + p.unit_eps), rk = 1.0f / sqrtf(rk + p.unit_eps);
    float seen = 0.f;
#pragma unroll
    for (int i = 0; i < ROWS; i += 4) {
      const float4 k4 = *reinterpret_cast<const float4*>(&ks[row0 + i]);
      s[i] *= g, s[i + 1] *= g, s[i + 2] *= g, s[i + 3] *= g;
      seen = fmaf(s[i], k4.x, fmaf(s[i + 1], k4.y, fmaf(s[i + 2], k4.z, fmaf(s[i + 3], k4.w, seen))));
    }
    part[rw][col] = seen;
    __syncthreads();
    seen = (part[0][col] + part[1][col]) + (part[2][col] + part[3][col]);
    const float u = col_ok ? beta * (vs[col] - seen * rk) * rk : 0.f;
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < ROWS; i += 4) {
      const float4 k4 = *reinterpret_cast<const float4*>(&ks[row0 + i]);
      const float4 q4 = *reinterpret_cast<const float4*>(&qs[row0 + i]);
      s[i] = fmaf(k4.x, u, s[i]), o = fmaf(s[i], q4.x, o);
      s[i + 1] = fmaf(k4.y, u, s[i + 1]), o = fmaf(s[i + 1], q4.y, o);
      s[i + 2] = fmaf(k4.z, u, s[i + 2]), o = fmaf(s[i + 2], q4.z, o);
      s[i + 3] = fmaf(k4.w, u, s[i + 3]), o = fmaf(s[i + 3], q4.w, o);
    }
    __syncthreads();  // everyone has read the first partial sums
    part[rw][col] = o;
    __syncthreads();
    o = ((part[0][col] + part[1][col]) + (part[2][col] + part[3][col])) * rq;
    // norm over the head: the first row group's warps hold every column once
    const float sq = warp_sum(rw == 0 && col_ok ? o * o : 0.f);
    if (lane == 0) red[2][warp] = sq;
    __syncthreads();
    if (rw == 0 && col_ok) {
      float total = 0.f;
      for (int i = 0; i < n_warps; i += kStepRowWarps) total += red[2][i];
      const float inv = 1.0f / sqrtf(total / (float)vdim + p.eps);
      static_cast<T*>(p.y)[row * p.ld_y + h * vdim + col] = from_float<T>(o * inv * p.norm_w[col] * to_float(src[p.off_g + h * vdim + col]));
    }
    // (qs, ks, vs are written again only after everyone has passed the last barrier; red[2] behind the next token's first)
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i)
    if (col_ok && row0 + i < dim) st[(int64_t)(row0 + i) * vdim] = s[i];
  if (p.n == 1 && p.conv_state && taps > 1) {
    // this token's inputs take a slot that no block reads in this step; a key head's channels are its first value head's to store
    const T* src = static_cast<const T*>(p.rows) + b * p.ld;
    T* dst = static_cast<T*>(p.conv_state) + (b * taps + start % taps) * p.conv_cols;
    for (int c = threadIdx.x; c < channels; c += blockDim.x) {
      if (c < 2 * dim && h % group) continue;
      const int64_t col_in = c < dim ? kv * dim + c : c < 2 * dim ? p.off_k + kv * dim + (c - dim) : p.off_v + h * vdim + (c - 2 * dim);
      dst[col_in] = src[col_in];
    }
  }
}

// ------------------------------------------------------------------ one token, the state through shared memory
// One block per (sequence, head).  The state is on its way into shared memory (asynchronous copies: several blocks per SM
// have theirs in flight) while the convolutions run; a warp takes every eighth row, a lane four columns of 128.
constexpr int kTokenThreads = 256, kTokenWarps = kTokenThreads / 32, kTokenMaxDim = 256;

template <typename T>
__global__ void __launch_bounds__(kTokenThreads)
delta_token_kernel(b200_delta_args p) {
  extern __shared__ __align__(16) float S[];  // [dim][vdim], then partial sums [warps][128]
  __shared__ float qs[kTokenMaxDim], ks[kTokenMaxDim], vs[kStepMaxCols], os[kStepMaxCols], red[2][kTokenWarps];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int dim = (int)p.dim, vdim = (int)p.vdim, taps = (int)p.taps;
  const int heads = (int)p.heads, h = (int)(blockIdx.x % heads), group = heads / (int)p.kv_heads, kv = h / group;
  const int64_t b = blockIdx.x / heads;
  const int start = p.pos_dev ? p.pos_dev[0] : (int)p.start;
  float* st = p.state + (b * heads + h) * (int64_t)dim * vdim;
  float* part = S + dim * vdim;
  for (int i = threadIdx.x; i < dim * vdim / 4; i += kTokenThreads)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(S + i * 4)), "l"(st + i * 4) : "memory");
  asm volatile("cp.async.commit_group;" ::: "memory");
  const T* src = static_cast<const T*>(p.rows) + b * p.ld;
  T* ring = static_cast<T*>(p.conv_state) + b * taps * p.conv_cols;
  const int slot = start % taps;  // this token's; the one before it is one slot down
  float sq_q = 0.f, sq_k = 0.f;
  for (int c = threadIdx.x; c < 2 * dim + vdim; c += kTokenThreads) {
    const int64_t col = c < dim ? (int64_t)kv * dim + c : c < 2 * dim ? p.off_k + kv * dim + (c - dim) : p.off_v + h * vdim + (c - 2 * dim);
    const float* w = p.conv_w + col * taps;
    const T now = src[col];
    float a = w[taps - 1] * to_float(now);
    for (int back = 1; back < taps; ++back)
      if (start >= back) a = fmaf(w[taps - 1 - back], to_float(ring[(int64_t)(slot >= back ? slot - back : slot - back + taps) * p.conv_cols + col]), a);
    // (no block reads this slot in this step; a key head's channels are its first value head's to store)
    if (taps > 1 && p.conv_state && (c >= 2 * dim || h % group == 0)) ring[(int64_t)slot * p.conv_cols + col] = now;
    const float o = to_float(from_float<T>(silu_exact(a)));
    if (c < dim) qs[c] = o, sq_q = fmaf(o, o, sq_q);
    else if (c < 2 * dim) ks[c - dim] = o, sq_k = fmaf(o, o, sq_k);
    else vs[c - 2 * dim] = o;
  }
  sq_q = warp_sum(sq_q), sq_k = warp_sum(sq_k);
  if (lane == 0) red[0][warp] = sq_q, red[1][warp] = sq_k;
  const float g = expf(-expf(p.a_log[h]) * softplus_exact(to_float(src[p.off_a + h]) + p.dt_bias[h]));
  const float beta = 1.0f / (1.0f + expf(-to_float(src[p.off_b + h])));
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  float rq = 0.f, rk = 0.f;
#pragma unroll
  for (int i = 0; i < kTokenWarps; ++i) rq += red[0][i], rk += red[1][i];
  rq = p.q_scale / sqrtf(rq + p.unit_eps), rk = 1.0f / sqrtf(rk + p.unit_eps);
  // a lane's four columns, summed over the warps' rows
  auto meet = [&](float4 x) -> float4 {
    __syncthreads();
    *reinterpret_cast<float4*>(part + warp * 128 + lane * 4) = x;
    __syncthreads();
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < kTokenWarps; ++i) {
      const float4 y = *reinterpret_cast<const float4*>(part + i * 128 + lane * 4);
      s.x += y.x, s.y += y.y, s.z += y.z, s.w += y.w;
    }
    return s;
  };
  float sq = 0.f;
  for (int c0 = 0; c0 < vdim; c0 += 128) {
    const int c = c0 + lane * 4;
    const bool ok = c < vdim;
    float4 seen = make_float4(0.f, 0.f, 0.f, 0.f);
    if (ok) {
#pragma unroll 4
      for (int r = warp; r < dim; r += kTokenWarps) {
        const float4 x = *reinterpret_cast<const float4*>(S + r * vdim + c);
        const float k = ks[r];
        seen.x = fmaf(x.x, k, seen.x), seen.y = fmaf(x.y, k, seen.y), seen.z = fmaf(x.z, k, seen.z), seen.w = fmaf(x.w, k, seen.w);
      }
    }
    seen = meet(seen);
    const float f = g * rk, bk = beta * rk;
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f), o = u;
    if (ok) {
      u = make_float4(bk * (vs[c] - f * seen.x), bk * (vs[c + 1] - f * seen.y), bk * (vs[c + 2] - f * seen.z), bk * (vs[c + 3] - f * seen.w));
#pragma unroll 4
      for (int r = warp; r < dim; r += kTokenWarps) {
        float4 x = *reinterpret_cast<const float4*>(S + r * vdim + c);
        const float k = ks[r], q = qs[r];
        x = make_float4(fmaf(k, u.x, g * x.x), fmaf(k, u.y, g * x.y), fmaf(k, u.z, g * x.z), fmaf(k, u.w, g * x.w));
        *reinterpret_cast<float4*>(st + (int64_t)r * vdim + c) = x;
        o.x = fmaf(x.x, q, o.x), o.y = fmaf(x.y, q, o.y), o.z = fmaf(x.z, q, o.z), o.w = fmaf(x.w, q, o.w);
      }
    }
    o = meet(o);
    o = make_float4(o.x * rq, o.y * rq, o.z * rq, o.w * rq);
    if (ok) {
      sq = fmaf(o.x, o.x, fmaf(o.y, o.y, fmaf(o.z, o.z, fmaf(o.w, o.w, sq))));
      if (warp == 0) *reinterpret_cast<float4*>(os + c) = o;
    }
  }
  const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)vdim + p.eps);  // (every warp holds all columns)
  __syncthreads();
  for (int c = threadIdx.x; c < vdim; c += kTokenThreads)
    static_cast<T*>(p.y)[b * p.ld_y + h * vdim + c] = from_float<T>(os[c] * inv * p.norm_w[c] * to_float(src[p.off_g + h * vdim + c]));
}

int token_smem(const b200_delta_args& p) { return (int)(p.dim * p.vdim + kTokenWarps * 128) * 4; }
bool takes_token(const b200_delta_args& p) {
  return p.n == 1 && !p.fresh && p.conv_state && p.dim <= kTokenMaxDim && p.vdim <= kStepMaxCols && p.vdim % 4 == 0 && token_smem(p) <= 200 * 1024 &&
         (reinterpret_cast<uintptr_t>(p.state) & 15) == 0 && p.start < 0x7fffffffLL;
}

template <typename T>
int launch_token(const b200_delta_args& p, cudaStream_t stream) {
  static std::atomic<bool> done[kMaxDevices];
  const int slot = device_slot();
  if (slot < 0) return B200_ERR_CUDA;
  if (!done[slot].load(std::memory_order_acquire)) {
    if (cudaFuncSetAttribute(delta_token_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return B200_ERR_CUDA;
    done[slot].store(true, std::memory_order_release);
  }
  delta_token_kernel<T><<<(unsigned)(p.B * p.heads), kTokenThreads, token_smem(p), stream>>>(p);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

bool takes_step(const b200_delta_args& p) {
  return p.dim <= 128 && p.vdim <= kStepMaxCols;
}

template <typename T>
int launch_step(const b200_delta_args& p, cudaStream_t stream) {
  const unsigned threads = 32 * kStepRowWarps * (unsigned)((p.vdim + 31) / 32), blocks = (unsigned)(p.B * p.heads);
  if (p.dim <= 64 && threads <= 512) delta_step_kernel<T, 16, 512><<<blocks, threads, 0, stream>>>(p);
  else if (p.dim <= 64) delta_step_kernel<T, 16, 1024><<<blocks, threads, 0, stream>>>(p);
  else if (threads <= 512) delta_step_kernel<T, 32, 512><<<blocks, threads, 0, stream>>>(p);
  else delta_step_kernel<T, 32, 1024><<<blocks, threads, 0, stream>>>(p);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

template <typename T>
int launch_store(const b200_delta_args& p, cudaStream_t stream) {
  if (!p.conv_state || p.taps < 2) return B200_OK;
  int64_t cols = (p.conv_cols + 255) / 256;
  if (cols > 64) cols = 64;
  conv_store_kernel<T><<<dim3((unsigned)p.B, (unsigned)cols), 256, 0, stream>>>(p);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

template <typename T>
int launch_typed(const b200_delta_args& p, cudaStream_t stream) {
  const int64_t tiles = (p.n + kInputTokens - 1) / kInputTokens;
  if (p.B > 65535 || p.B * tiles > 0x7fffffffLL || p.B * p.heads > 0x7fffffffLL) return B200_ERR_BAD_ARGUMENT;
  int st = B200_OK;
  if (delta_chunk_takes(p)) {
    st = launch_delta_chunk(p, stream);
  } else if (takes_token(p)) {
    return launch_token<T>(p, stream);
  } else if (takes_step(p)) {
    st = launch_step<T>(p, stream);
    if (p.n == 1) return st;
  } else {
    const size_t smem = (size_t)(2 * p.dim + p.vdim) * 4;
    if (smem > 47 * 1024) return B200_ERR_UNSUPPORTED;
    delta_inputs_kernel<T><<<(unsigned)(p.B * tiles), 32 * kInputWarps, 0, stream>>>(p, tiles);
    delta_any_kernel<T><<<(unsigned)(p.B * p.heads), kAnyThreads, smem, stream>>>(p);
    note_launches(2);
    st = status_from_cuda(cudaGetLastError());
  }
  return st == B200_OK ? launch_store<T>(p, stream) : st;
}

}  // namespace

int64_t delta_workspace_bytes(const b200_delta_args& p) { return delta_chunk_takes(p) ? delta_chunk_workspace_bytes(p) : 0; }

int launch_delta(const b200_delta_args& p, cudaStream_t stream) {
  return p.dtype == B200_BF16 ? launch_typed<__nv_bfloat16>(p, stream) : launch_typed<float>(p, stream);
}

}  // namespace b200
