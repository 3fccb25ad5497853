// Queries and keys behind their products: RMS norm per head, rotation of the first columns of a head by the token's position,
// and keys and values into the rows that attention reads and into the ring that remembers them.
#include "common.cuh"

namespace b200 {
namespace {

constexpr int kTokenWarps = 8;
constexpr int kMaxPairs = 8;        // column pairs per lane: heads of up to 512 columns
constexpr int kMaxRotPairs = 256;

// sin and cos of pos * f with f = f_hi + f_lo: the product is exact to twice fp32's precision, so that the angle carries no
// rounding that grows with the position.
__device__ __forceinline__ float2 position_angle(float pos, float f_hi, float f_lo) {
  const float a = pos * f_hi;
  const float rest = fmaf(pos, f_hi, -a) + pos * f_lo;
  float s, c;
  sincosf(a, &s, &c);
  const float r2 = rest * rest;  // (|rest| is at most half a unit in the last place of a)
  const float cr = fmaf(r2, fmaf(r2, 1.0f / 24.0f, -0.5f), 1.0f), sr = rest * fmaf(r2, -1.0f / 6.0f, 1.0f);
  return make_float2(c * cr - s * sr, s * cr + c * sr);  // (cos, sin)
}

template <typename T>
__device__ __forceinline__ void store_value(void* dst, int64_t at, float v, int dtype) {
  if (dtype == B200_F16) static_cast<__half*>(dst)[at] = __float2half_rn(v);
  else static_cast<T*>(dst)[at] = from_float<T>(v);
}

// One block per token; a warp takes one head at a time.  rows: q heads | k heads | v heads, sections at columns off_*.
template <typename T>
__global__ void __launch_bounds__(32 * kTokenWarps)
rotary_kernel(b200_rotary_args p) {
  __shared__ float2 turn[kMaxRotPairs];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t row = blockIdx.x, b = row / p.n, t = row % p.n;
  const int64_t pos = (p.pos_dev ? (int64_t)p.pos_dev[0] : p.start) + t;
  const int rot_pairs = (int)p.rot_dims / 2;
  for (int i = threadIdx.x; i < rot_pairs; i += 32 * kTokenWarps) turn[i] = position_angle((float)pos, p.freq[2 * i], p.freq[2 * i + 1]);
  __syncthreads();
  const int dim = (int)p.dim, pairs = (dim + 1) / 2;
  const int64_t work_row = b * (p.hist + p.n) + p.hist + t;
  const bool keep = p.k_cache && t + p.ring >= p.n && pos >= 0;
  const int64_t slot = keep ? pos % p.ring : 0;
  T* rows = static_cast<T*>(p.rows) + row * p.ld;
  const int key_maps = (int)(p.kv_heads * p.maps);
  for (int head = warp; head < (int)p.q_heads + key_maps; head += kTokenWarps) {
    const bool is_q = head < (int)p.q_heads;
    const int k_index = head - (int)p.q_heads;
    T* src = rows + (is_q ? (int64_t)head * dim : p.off_k + (int64_t)k_index * dim);
    const float* w = is_q ? p.q_weight : p.k_weight;
    float u[kMaxPairs], v[kMaxPairs], s = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxPairs; ++i) {
      const int c = 2 * (i * 32 + lane);
      u[i] = c < dim ? to_float(src[c]) : 0.f;
      v[i] = c + 1 < dim ? to_float(src[c + 1]) : 0.f;
      s = fmaf(u[i], u[i], fmaf(v[i], v[i], s));
      if ((i + 1) * 32 >= pairs) break;
    }
    const float inv = 1.0f / sqrtf(warp_sum(s) / (float)dim + p.eps);
#pragma unroll
    for (int i = 0; i < kMaxPairs; ++i) {
      const int pi = i * 32 + lane, c = 2 * pi;
      if (c < dim) {
        float a = u[i] * inv * w[c], z = c + 1 < dim ? v[i] * inv * w[c + 1] : 0.f;
        if (pi < rot_pairs) {
          const float2 cs = turn[pi];
          const float ra = a * cs.x - z * cs.y;
          z = z * cs.x + a * cs.y;
          a = ra;
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (c + e >= dim) break;
          const T o = from_float<T>(e ? z : a);
          if (is_q) {
            src[c + e] = o;
          } else {
            if (p.k_rows) static_cast<T*>(p.k_rows)[work_row * p.ld_k + (int64_t)k_index * dim + c + e] = o;
            if (keep) {
              const int64_t g = k_index / p.maps, m = k_index % p.maps;
              static_cast<T*>(p.k_cache)[((b * p.kv_heads + g) * p.ring + slot) * (p.maps * dim) + m * dim + c + e] = o;
            }
          }
        }
      }
      if ((i + 1) * 32 >= pairs) break;
    }
  }
  const int64_t vcols = p.kv_heads * p.vdim;
  for (int64_t c = threadIdx.x; c < vcols; c += 32 * kTokenWarps) {
    const float f = to_float(rows[p.off_v + c]);
    if (p.v_rows) store_value<T>(p.v_rows, work_row * p.ld_v + c, f, p.v_rows_dtype);
    if (keep) static_cast<T*>(p.v_cache)[((b * p.kv_heads + c / p.vdim) * p.ring + slot) * p.vdim + c % p.vdim] = from_float<T>(f);
  }
}

// The same for heads of a multiple of 8 columns, up to 256: a lane takes 8 columns, the `lanes` (a power of two) lanes of a head
// sit side by side, and a block takes a few tokens.
constexpr int kMaxVecTokens = 4;
template <typename T>
__global__ void __launch_bounds__(32 * kTokenWarps)
rotary_vec_kernel(b200_rotary_args p, int lanes, int tokens) {
  __shared__ float2 turn[kMaxVecTokens][128];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t row0 = (int64_t)blockIdx.x * tokens, rows_total = p.B * p.n;
  const int nt = (int)(rows_total - row0 < tokens ? rows_total - row0 : tokens);
  const int rot_pairs = (int)p.rot_dims / 2, dim = (int)p.dim, vdim = (int)p.vdim;
  const int64_t first = p.pos_dev ? (int64_t)p.pos_dev[0] : p.start;
  for (int i = threadIdx.x; i < nt * rot_pairs; i += 32 * kTokenWarps) {
    const int t = i / rot_pairs, j = i % rot_pairs;
    turn[t][j] = position_angle((float)(first + (row0 + t) % p.n), p.freq[2 * j], p.freq[2 * j + 1]);
  }
  __syncthreads();
  const int per_warp = 32 / lanes, sub = lane / lanes, c = (lane % lanes) * 8;
  const int heads = (int)(p.q_heads + p.kv_heads * p.maps), groups = (heads + per_warp - 1) / per_warp;
  const float inv_dim = 1.0f / (float)dim;
  for (int item = warp; item < nt * groups; item += kTokenWarps) {
    const int tt = item / groups, head = item % groups * per_warp + sub;
    const int64_t row = row0 + tt, b = row / p.n, t = row % p.n, pos = first + t;
    const bool ok = head < heads && c < dim, is_q = head < (int)p.q_heads;
    const int ki = head - (int)p.q_heads;
    T* src = static_cast<T*>(p.rows) + row * p.ld + (is_q ? (int64_t)head * dim : p.off_k + (int64_t)ki * dim) + c;
    float f[8], w[8], s = 0.f;
    if (ok) {
      load8(src, f);
      load8((is_q ? p.q_weight : p.k_weight) + c, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) s = fmaf(f[e], f[e], s);
    }
    for (int o = 1; o < lanes; o <<= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (!ok) continue;
    const float inv = 1.0f / sqrtf(s * inv_dim + p.eps);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] *= inv * w[e];
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      const int pi = (c + e) / 2;
      if (pi < rot_pairs) {
        const float2 cs = turn[tt][pi];
        const float u = f[e], v = f[e + 1];
        f[e] = u * cs.x - v * cs.y;
        f[e + 1] = v * cs.x + u * cs.y;
      }
    }
    if (is_q) {
      store8(src, f);
    } else {
      if (p.k_rows) store8(static_cast<T*>(p.k_rows) + (b * (p.hist + p.n) + p.hist + t) * p.ld_k + (int64_t)ki * dim + c, f);
      if (p.k_cache && t + p.ring >= p.n) {
        const int64_t g = ki / p.maps, m = ki % p.maps;
        store8(static_cast<T*>(p.k_cache) + ((b * p.kv_heads + g) * p.ring + pos % p.ring) * (p.maps * dim) + m * dim + c, f);
      }
    }
  }
  const int vecs = (int)(p.kv_heads * vdim) / 8;
  for (int i = threadIdx.x; i < nt * vecs; i += 32 * kTokenWarps) {
    const int tt = i / vecs;
    const int64_t vc = (int64_t)(i % vecs) * 8, row = row0 + tt, b = row / p.n, t = row % p.n;
    float f[8];
    load8(static_cast<const T*>(p.rows) + row * p.ld + p.off_v + vc, f);
    const int64_t work_row = b * (p.hist + p.n) + p.hist + t;
    if (p.v_rows) {
      if (p.v_rows_dtype == B200_F16) store8(static_cast<__half*>(p.v_rows) + work_row * p.ld_v + vc, f);
      else store8(static_cast<T*>(p.v_rows) + work_row * p.ld_v + vc, f);
    }
    if (p.k_cache && t + p.ring >= p.n)
      store8(static_cast<T*>(p.v_cache) + ((b * p.kv_heads + vc / vdim) * p.ring + (first + t) % p.ring) * vdim + vc % vdim, f);
  }
}

// Rows [0, hist) of k_rows and v_rows: what the ring remembers of the positions [start - hist, start).
template <typename T>
__global__ void __launch_bounds__(256)
ring_gather_kernel(b200_rotary_args p) {
  const int64_t b = blockIdx.x / p.hist, j = blockIdx.x % p.hist;
  const int64_t slot = (p.start - p.hist + j) % p.ring, work_row = b * (p.hist + p.n) + j;
  const int64_t kd = p.maps * p.dim;
  for (int64_t c = threadIdx.x; c < p.kv_heads * kd; c += 256)
    static_cast<T*>(p.k_rows)[work_row * p.ld_k + c] = static_cast<const T*>(p.k_cache)[((b * p.kv_heads + c / kd) * p.ring + slot) * kd + c % kd];
  for (int64_t c = threadIdx.x; c < p.kv_heads * p.vdim; c += 256)
    store_value<T>(p.v_rows, work_row * p.ld_v + c,
                   to_float(static_cast<const T*>(p.v_cache)[((b * p.kv_heads + c / p.vdim) * p.ring + slot) * p.vdim + c % p.vdim]), p.v_rows_dtype);
}

template <typename T>
int launch_typed(const b200_rotary_args& p, cudaStream_t stream) {
  if (p.dim > 64 * kMaxPairs || p.rot_dims > 2 * kMaxRotPairs) return B200_ERR_UNSUPPORTED;
  if (p.hist) {
    ring_gather_kernel<T><<<(unsigned)(p.B * p.hist), 256, 0, stream>>>(p);
    note_launches(1);
  }
  const uintptr_t al = reinterpret_cast<uintptr_t>(p.rows) | reinterpret_cast<uintptr_t>(p.q_weight) | reinterpret_cast<uintptr_t>(p.k_weight) |
                       reinterpret_cast<uintptr_t>(p.k_rows) | reinterpret_cast<uintptr_t>(p.v_rows) | reinterpret_cast<uintptr_t>(p.k_cache) |
                       reinterpret_cast<uintptr_t>(p.v_cache);
  const bool pitches = p.ld % 8 == 0 && p.off_k % 8 == 0 && p.off_v % 8 == 0 && (!p.k_rows || (p.ld_k % 8 == 0 && p.ld_v % 8 == 0));
  if ((al & 15) == 0 && pitches && p.dim % 8 == 0 && p.vdim % 8 == 0 && p.dim <= 256) {
    int lanes = 1;
    while (lanes * 8 < p.dim) lanes *= 2;
    const int64_t rows = p.B * p.n;
    const int tokens = rows >= 4096 ? kMaxVecTokens : 1;
    rotary_vec_kernel<T><<<(unsigned)((rows + tokens - 1) / tokens), 32 * kTokenWarps, 0, stream>>>(p, lanes, tokens);
  } else {
    rotary_kernel<T><<<(unsigned)(p.B * p.n), 32 * kTokenWarps, 0, stream>>>(p);
  }
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

}  // namespace

int launch_rotary_append(const b200_rotary_args& p, cudaStream_t stream) {
  return p.dtype == B200_BF16 ? launch_typed<__nv_bfloat16>(p, stream) : launch_typed<float>(p, stream);
}

}  // namespace b200
