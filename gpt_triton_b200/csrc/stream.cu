// One pass over the rows of an fp32 residual stream between two sublayers: whatever is added to the stream (a sublayer's
// output behind a norm of its own, token embeddings, one vector for all rows) and the norm in front of the next sublayer.
#include "common.cuh"

namespace b200 {
namespace {

constexpr int kMaxThreads = 256;

__device__ __forceinline__ float block_sum(float v, float* part) {
  v = warp_sum(v);
  if (blockDim.x == 32) return v;
  __syncthreads();  // (the previous sum has been read)
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (unsigned i = 0; i < blockDim.x / 32; ++i) s += part[i];
  return s;
}

// One block per row; NV vectors of 8 elements per thread stay in registers from the load to the store.
template <typename T, int NV>
__global__ void __launch_bounds__(kMaxThreads)
stream_update_kernel(b200_stream_args p) {
  __shared__ float part[kMaxThreads / 32];
  const int64_t t = blockIdx.x;
  const int W = (int)p.W;
  float* xr = p.x + t * W;
  float v[NV][8];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * 8;
#pragma unroll
    for (int e = 0; e < 8; ++e) v[i][e] = 0.f;
    if (p.keep && c < W) load8(xr + c, v[i]);
  }
  if (p.y) {
    const T* yr = static_cast<const T*>(p.y) + t * p.ld_y;
    float f[NV][8], s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * (int)blockDim.x + (int)threadIdx.x) * 8;
      if (c < W) {
        load8(yr + c, f[i]);
#pragma unroll
        for (int e = 0; e < 8; ++e) s = fmaf(f[i][e], f[i][e], s);
      }
    }
    const float inv = 1.0f / sqrtf(block_sum(s, part) / (float)W + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * (int)blockDim.x + (int)threadIdx.x) * 8;
      if (c < W) {
        float g[8];
        load8(p.y_gain + c, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] = fmaf(f[i][e] * inv, g[e], v[i][e]);
      }
    }
  }
  const int64_t id = p.ids ? p.ids[t] : -1;
  const bool add_table = id >= 0 && id < p.V;
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * 8;
    if (c < W) {
      float f[8];
      if (add_table) {
        load8(static_cast<const T*>(p.table) + id * W + c, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] += f[e] * p.table_scale;
      }
      if (p.shift) {
        load8(p.shift + c, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] += f[e];
      }
      store8(xr + c, v[i]);
#pragma unroll
      for (int e = 0; e < 8; ++e) s = fmaf(v[i][e], v[i][e], s);
    }
  }
  if (!p.gain) return;
  const float inv = 1.0f / sqrtf(block_sum(s, part) / (float)W + p.eps);
  T* hr = static_cast<T*>(p.h) + t * p.ld_h;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * 8;
    if (c < W) {
      float g[8];
      load8(p.gain + c, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) g[e] *= v[i][e] * inv;
      store8(hr + c, g);
    }
  }
}

// Any width and alignment: the row is read again for every step.
template <typename T>
__global__ void __launch_bounds__(kMaxThreads)
stream_update_any_kernel(b200_stream_args p) {
  __shared__ float part[kMaxThreads / 32];
  const int64_t t = blockIdx.x;
  float* xr = p.x + t * p.W;
  const T* yr = p.y ? static_cast<const T*>(p.y) + t * p.ld_y : nullptr;
  float y_inv = 0.f;
  if (yr) {
    float s = 0.f;
    for (int64_t c = threadIdx.x; c < p.W; c += blockDim.x) {
      const float f = to_float(yr[c]);
      s = fmaf(f, f, s);
    }
    y_inv = 1.0f / sqrtf(block_sum(s, part) / (float)p.W + p.eps);
  }
  const int64_t id = p.ids ? p.ids[t] : -1;
  const T* row = id >= 0 && id < p.V ? static_cast<const T*>(p.table) + id * p.W : nullptr;
  float s = 0.f;
  for (int64_t c = threadIdx.x; c < p.W; c += blockDim.x) {
    float v = p.keep ? xr[c] : 0.f;
    if (yr) v = fmaf(to_float(yr[c]) * y_inv, p.y_gain[c], v);
    if (row) v += to_float(row[c]) * p.table_scale;
    if (p.shift) v += p.shift[c];
    xr[c] = v;
    s = fmaf(v, v, s);
  }
  if (!p.gain) return;
  const float inv = 1.0f / sqrtf(block_sum(s, part) / (float)p.W + p.eps);
  T* hr = static_cast<T*>(p.h) + t * p.ld_h;
  for (int64_t c = threadIdx.x; c < p.W; c += blockDim.x) hr[c] = from_float<T>(xr[c] * inv * p.gain[c]);
}

// One thread per 8 outputs; columns of z in blocks of 64: 32 gates, then their 32 ups.
template <typename T>
__global__ void __launch_bounds__(256)
gated_pairs_kernel(const T* __restrict__ z, int64_t ld_z, T* __restrict__ out, int64_t ld_out, int64_t T_, int64_t F, float limit, float alpha) {
  const int64_t per_row = (F + 7) / 8, i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (i >= T_ * per_row) return;
  const int64_t t = i / per_row, c = (i % per_row) * 8;
  const T* src = z + t * ld_z + c / 32 * 64 + c % 32;
  for (int e = 0; e < 8 && c + e < F; ++e) {
    const float g = fminf(to_float(src[e]), limit), u = fminf(fmaxf(to_float(src[e + 32]), -limit), limit);
    out[t * ld_out + c + e] = from_float<T>(g / (1.0f + expf(-alpha * g)) * (u + 1.0f));
  }
}

template <typename T>
int launch_typed(const b200_stream_args& p, cudaStream_t stream) {
  const uintptr_t al = reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.y) | reinterpret_cast<uintptr_t>(p.y_gain) |
                       reinterpret_cast<uintptr_t>(p.table) | reinterpret_cast<uintptr_t>(p.shift) | reinterpret_cast<uintptr_t>(p.gain) |
                       reinterpret_cast<uintptr_t>(p.h);
  const bool vec = (al & 15) == 0 && p.W % 8 == 0 && (!p.y || p.ld_y % 8 == 0) && (!p.gain || p.ld_h % 8 == 0);
  const unsigned grid = (unsigned)p.T;
  int64_t threads = (p.W / 8 + 31) / 32 * 32;
  if (threads > kMaxThreads) threads = kMaxThreads;
  if (threads < 32) threads = 32;
  const int64_t nv = (p.W / 8 + threads - 1) / threads;
  if (vec && nv <= 1) stream_update_kernel<T, 1><<<grid, (unsigned)threads, 0, stream>>>(p);
  else if (vec && nv <= 2) stream_update_kernel<T, 2><<<grid, (unsigned)threads, 0, stream>>>(p);
  else if (vec && nv <= 4) stream_update_kernel<T, 4><<<grid, (unsigned)threads, 0, stream>>>(p);
  else stream_update_any_kernel<T><<<grid, kMaxThreads, 0, stream>>>(p);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

}  // namespace

int launch_gated_pairs(const void* z, int64_t ld_z, void* out, int64_t ld_out, int64_t T, int64_t F, float limit, float alpha, int dtype, cudaStream_t stream) {
  const int64_t blocks = (T * ((F + 7) / 8) + 255) / 256;
  if (blocks > 0x7fffffffLL) return B200_ERR_BAD_ARGUMENT;
  if (dtype == B200_BF16)
    gated_pairs_kernel<<<(unsigned)blocks, 256, 0, stream>>>((const __nv_bfloat16*)z, ld_z, (__nv_bfloat16*)out, ld_out, T, F, limit, alpha);
  else
    gated_pairs_kernel<<<(unsigned)blocks, 256, 0, stream>>>((const float*)z, ld_z, (float*)out, ld_out, T, F, limit, alpha);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

int launch_stream_update(const b200_stream_args& p, cudaStream_t stream) {
  return p.dtype == B200_BF16 ? launch_typed<__nv_bfloat16>(p, stream) : launch_typed<float>(p, stream);
}

}  // namespace b200
