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
  rotary_kernel<T><<<(unsigned)(p.B * p.n), 32 * kTokenWarps, 0, stream>>>(p);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

}  // namespace

int launch_rotary_append(const b200_rotary_args& p, cudaStream_t stream) {
  return p.dtype == B200_BF16 ? launch_typed<__nv_bfloat16>(p, stream) : launch_typed<float>(p, stream);
}

}  // namespace b200
