// Latent attention: the per-token latent cache, sliding-window attention with a sink over expanded keys and values (a
// prompt or a portion of one), and one-token decoding straight on the cached latents.  The kernels of this file take any
// sizes and both storage types; fp32 storage is computed in true 32-bit throughout.
#include "common.cuh"

namespace b200 {
namespace {

// ------------------------------------------------------------------ latents in and out of the cache
// One warp per new token: RMS norm over R, then to the work rows and, for the last `ring` tokens, to the cache.  VEC: rows
// of up to 1024 elements move as 8-element vectors and stay in registers.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
latent_append_kernel(const T* __restrict__ raw, int64_t ld_raw, const float* __restrict__ weight, float eps, T* __restrict__ work,
                     T* __restrict__ cache, int64_t rows, int64_t n_new, int64_t R, int64_t hist, int64_t ring, int64_t start,
                     const int* __restrict__ pos_dev) {
  const int lane = threadIdx.x & 31;
  const int64_t row = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (row >= rows) return;
  const int64_t b = row / n_new, t = row % n_new;
  const int64_t pos = (pos_dev ? (int64_t)pos_dev[0] : start) + t;
  const T* src = raw + row * ld_raw;
  if constexpr (VEC) {
    constexpr int NV = 4;
    T* w = work ? work + (b * (hist + n_new) + hist + t) * R : nullptr;
    T* k = (cache && t + ring >= n_new && pos >= 0) ? cache + (b * ring + pos % ring) * R : nullptr;
    float f[NV][8], s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * 32 + lane) * 8;
      if (c < R) {
        load8(src + c, f[i]);
#pragma unroll
        for (int e = 0; e < 8; ++e) s = fmaf(f[i][e], f[i][e], s);
      }
    }
    const float inv = 1.0f / sqrtf(warp_sum(s) / (float)R + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * 32 + lane) * 8;
      if (c < R) {
        float g[8];
        load8(weight + c, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) g[e] *= f[i][e] * inv;
        if (w) store8(w + c, g);
        if (k) store8(k + c, g);
      }
    }
    return;
  }
  float s = 0.f;
  for (int64_t c = lane; c < R; c += 32) {
    const float v = to_float(src[c]);
    s = fmaf(v, v, s);
  }
  const float inv = 1.0f / sqrtf(warp_sum(s) / (float)R + eps);
  T* w = work ? work + (b * (hist + n_new) + hist + t) * R : nullptr;
  T* k = (cache && t + ring >= n_new && pos >= 0) ? cache + (b * ring + pos % ring) * R : nullptr;
  for (int64_t c = lane; c < R; c += 32) {
    const T v = from_float<T>(to_float(src[c]) * inv * weight[c]);
    if (w) w[c] = v;
    if (k) k[c] = v;
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
latent_gather_kernel(const T* __restrict__ cache, T* __restrict__ work, int64_t rows, int64_t n_new, int64_t R, int64_t hist, int64_t ring,
                     int64_t start) {
  const int lane = threadIdx.x & 31;
  const int64_t row = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (row >= rows) return;
  const int64_t b = row / hist, j = row % hist;
  const T* src = cache + (b * ring + (start - hist + j) % ring) * R;
  T* dst = work + (b * (hist + n_new) + j) * R;
  for (int64_t c = lane; c < R; c += 32) dst[c] = src[c];
}

// ------------------------------------------------------------------ sliding-window attention, any sizes
// One warp per query; 32 keys at a time, one per lane, online softmax; the output row lives in shared memory (a lane
// owns every 32nd column, so nothing needs a barrier).
constexpr int kQueryWarps = 4;
template <typename T>
__global__ void __launch_bounds__(32 * kQueryWarps)
window_attention_kernel(const T* __restrict__ q, int64_t ld_q, const T* __restrict__ k, int64_t ld_k, const T* __restrict__ v, int64_t ld_v,
                        T* __restrict__ out, int64_t ld_out, int64_t n_queries, int64_t n_new, int64_t hist, int64_t heads, int64_t dim,
                        int64_t vdim, int64_t window, float scale, const float* __restrict__ sink) {
  extern __shared__ float smem_f[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* qs = smem_f + warp * (dim + vdim);
  float* o = qs + dim;
  const int64_t item = (int64_t)blockIdx.x * kQueryWarps + warp;
  if (item >= n_queries) return;
  const int64_t h = item % heads, row = item / heads, b = row / n_new, t = row % n_new;
  for (int64_t c = lane; c < dim; c += 32) qs[c] = to_float(q[row * ld_q + h * dim + c]);
  for (int64_t c = lane; c < vdim; c += 32) o[c] = 0.f;
  __syncwarp();
  const int64_t last = hist + t, first = last + 1 > window ? last + 1 - window : 0;
  const int64_t kv0 = b * (hist + n_new);
  float m = -INFINITY, l = 0.f;
  for (int64_t j0 = first; j0 <= last; j0 += 32) {
    const int64_t j = j0 + lane;
    float s = -INFINITY;
    if (j <= last) {
      const T* kr = k + (kv0 + j) * ld_k + h * dim;
      float a = 0.f;
      for (int64_t c = 0; c < dim; ++c) a = fmaf(qs[c], to_float(kr[c]), a);
      s = a * scale;
    }
    float mb = s;
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mb = fmaxf(mb, __shfl_xor_sync(0xffffffffu, mb, off));
    const float m_new = fmaxf(m, mb);
    const float mult = expf(m - m_new);
    const float p = expf(s - m_new);
    l = l * mult + warp_sum(p);
    m = m_new;
    const int n = (int)(last - j0 + 1 < 32 ? last - j0 + 1 : 32);
    for (int64_t c0 = 0; c0 < vdim; c0 += 32) {
      const int64_t c = c0 + lane;
      float a = c < vdim ? o[c] * mult : 0.f;
      const T* vr = v + (kv0 + j0) * ld_v + h * vdim + c;
      for (int i = 0; i < n; ++i) {
        const float pi = __shfl_sync(0xffffffffu, p, i);
        if (c < vdim) a = fmaf(pi, to_float(vr[(int64_t)i * ld_v]), a);
      }
      if (c < vdim) o[c] = a;
    }
  }
  if (sink) l += expf(sink[h] - m);  // (inf if the sink dwarfs every score: the weights are then 0, as they should be)
  for (int64_t c = lane; c < vdim; c += 32) out[row * ld_out + h * vdim + c] = from_float<T>(o[c] / l);
}

// ------------------------------------------------------------------ decoding on the latents, any sizes
constexpr int kBatchTile = 8;
// q~[b, h, r] = sum_d q[b, h, d] * w_uk[h, d, r]; a thread owns r for up to kBatchTile sequences.
template <typename T>
__global__ void __launch_bounds__(128)
absorb_query_kernel(const T* __restrict__ q, int64_t ld_q, const T* __restrict__ w_uk, float* __restrict__ qt, int64_t B, int64_t heads,
                    int64_t dim, int64_t R) {
  const int64_t r = (int64_t)blockIdx.x * 128 + threadIdx.x, h = blockIdx.y, b0 = (int64_t)blockIdx.z * kBatchTile;
  if (r >= R) return;
  float acc[kBatchTile] = {};
  for (int64_t d = 0; d < dim; ++d) {
    const float w = to_float(w_uk[(h * dim + d) * R + r]);
#pragma unroll
    for (int i = 0; i < kBatchTile; ++i)
      if (b0 + i < B) acc[i] = fmaf(to_float(q[(b0 + i) * ld_q + h * dim + d]), w, acc[i]);
  }
#pragma unroll
  for (int i = 0; i < kBatchTile; ++i)
    if (b0 + i < B) qt[((b0 + i) * heads + h) * R + r] = acc[i];
}

// One block per (sequence, head): 64 latents at a time, online softmax, weighted latent sum o~[b, h, r] (normalised).
template <typename T>
__global__ void __launch_bounds__(128)
latent_decode_kernel(const float* __restrict__ qt, const T* __restrict__ cache, float* __restrict__ ot, int64_t heads, int64_t R, int64_t ring,
                     int64_t window, float scale, const float* __restrict__ sink, const int* __restrict__ pos_dev) {
  extern __shared__ float smem_f[];
  float* qs = smem_f;
  float* o = qs + R;
  float* sc = o + R;  // [64]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t h = blockIdx.x % heads, b = blockIdx.x / heads;
  const int64_t pos = pos_dev[0];
  const int64_t first = pos + 1 > window ? pos + 1 - window : 0;
  for (int64_t c = threadIdx.x; c < R; c += 128) qs[c] = qt[blockIdx.x * R + c], o[c] = 0.f;
  __syncthreads();
  float m = -INFINITY, l = 0.f;
  for (int64_t j0 = first; j0 <= pos; j0 += 64) {
    const int n = (int)(pos - j0 + 1 < 64 ? pos - j0 + 1 : 64);
    for (int i = warp; i < n; i += 4) {
      const T* c = cache + (b * ring + (j0 + i) % ring) * R;
      float a = 0.f;
      for (int64_t r = lane; r < R; r += 32) a = fmaf(qs[r], to_float(c[r]), a);
      a = warp_sum(a);
      if (lane == 0) sc[i] = a * scale;
    }
    __syncthreads();
    float m_new = m;
    for (int i = 0; i < n; ++i) m_new = fmaxf(m_new, sc[i]);
    const float mult = expf(m - m_new);
    m = m_new;
    __syncthreads();
    if (threadIdx.x < n) sc[threadIdx.x] = expf(sc[threadIdx.x] - m);
    __syncthreads();
    float ps = 0.f;
    for (int i = 0; i < n; ++i) ps += sc[i];
    l = l * mult + ps;
    for (int64_t r = threadIdx.x; r < R; r += 128) {
      float a = o[r] * mult;
      for (int i = 0; i < n; ++i) a = fmaf(sc[i], to_float(cache[(b * ring + (j0 + i) % ring) * R + r]), a);
      o[r] = a;
    }
    __syncthreads();
  }
  if (sink) l += expf(sink[h] - m);
  for (int64_t r = threadIdx.x; r < R; r += 128) ot[blockIdx.x * R + r] = o[r] / l;
}

// out[b, h, v] = sum_r w_uv[h, v, r] * o~[b, h, r]; a warp owns (h, v) for up to kBatchTile sequences.
template <typename T>
__global__ void __launch_bounds__(128)
expand_value_kernel(const float* __restrict__ ot, const T* __restrict__ w_uv, T* __restrict__ out, int64_t ld_out, int64_t B, int64_t heads,
                    int64_t vdim, int64_t R) {
  const int lane = threadIdx.x & 31;
  const int64_t hv = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5), b0 = (int64_t)blockIdx.y * kBatchTile;
  if (hv >= heads * vdim) return;
  const int64_t h = hv / vdim;
  float acc[kBatchTile] = {};
  for (int64_t r = lane; r < R; r += 32) {
    const float w = to_float(w_uv[hv * R + r]);
#pragma unroll
    for (int i = 0; i < kBatchTile; ++i)
      if (b0 + i < B) acc[i] = fmaf(ot[((b0 + i) * heads + h) * R + r], w, acc[i]);
  }
#pragma unroll
  for (int i = 0; i < kBatchTile; ++i) {
    const float s = warp_sum(acc[i]);
    if (lane == 0 && b0 + i < B) out[(b0 + i) * ld_out + hv] = from_float<T>(s);
  }
}

template <typename T>
int decode_typed(const void* q, int64_t ld_q, const void* w_uk, const void* w_uv, const void* cache, void* out, int64_t ld_out, int64_t B,
                 int64_t heads, int64_t dim, int64_t vdim, int64_t R, int64_t ring, int64_t window, float scale, const float* sink,
                 const int* pos_dev, void* workspace, cudaStream_t stream) {
  float* qt = static_cast<float*>(workspace);
  float* ot = qt + B * heads * R;
  const unsigned bt = (unsigned)((B + kBatchTile - 1) / kBatchTile);
  absorb_query_kernel<T><<<dim3((unsigned)((R + 127) / 128), (unsigned)heads, bt), 128, 0, stream>>>((const T*)q, ld_q, (const T*)w_uk, qt, B, heads, dim, R);
  const size_t smem = (size_t)(2 * R + 64) * 4;
  if (smem > 48 * 1024) return B200_ERR_UNSUPPORTED;
  latent_decode_kernel<T><<<(unsigned)(B * heads), 128, smem, stream>>>(qt, (const T*)cache, ot, heads, R, ring, window, scale, sink, pos_dev);
  expand_value_kernel<T><<<dim3((unsigned)((heads * vdim + 3) / 4), bt), 128, 0, stream>>>(ot, (const T*)w_uv, (T*)out, ld_out, B, heads, vdim, R);
  note_launches(3);
  return status_from_cuda(cudaGetLastError());
}

template <typename T>
int window_typed(const void* q, int64_t ld_q, const void* k, int64_t ld_k, const void* v, int64_t ld_v, void* out, int64_t ld_out, int64_t B,
                 int64_t n_new, int64_t hist, int64_t heads, int64_t dim, int64_t vdim, int64_t window, float scale, const float* sink,
                 cudaStream_t stream) {
  const int64_t n = B * n_new * heads, blocks = (n + kQueryWarps - 1) / kQueryWarps;
  const size_t smem = (size_t)kQueryWarps * (dim + vdim) * 4;
  if (smem > 48 * 1024 || blocks > 0x7fffffffLL) return B200_ERR_UNSUPPORTED;
  window_attention_kernel<T><<<(unsigned)blocks, 32 * kQueryWarps, smem, stream>>>((const T*)q, ld_q, (const T*)k, ld_k, (const T*)v, ld_v, (T*)out, ld_out,
                                                                                   n, n_new, hist, heads, dim, vdim, window, scale, sink);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

}  // namespace

template <typename T>
static int append_typed(const void* raw, int64_t ld_raw, const float* weight, float eps, void* work, void* cache, int64_t B, int64_t n_new, int64_t R,
                        int64_t hist, int64_t ring, int64_t start, const int* pos_dev, cudaStream_t stream) {
  const int64_t rows = B * n_new, blocks = (rows + 7) / 8;
  if (blocks > 0x7fffffffLL) return B200_ERR_BAD_ARGUMENT;
  const bool vec = R <= 1024 && R % 8 == 0 && ld_raw % 8 == 0 &&
                   ((reinterpret_cast<uintptr_t>(raw) | reinterpret_cast<uintptr_t>(weight) | reinterpret_cast<uintptr_t>(work) | reinterpret_cast<uintptr_t>(cache)) & 15) == 0;
  if (vec)
    latent_append_kernel<T, true><<<(unsigned)blocks, 256, 0, stream>>>((const T*)raw, ld_raw, weight, eps, (T*)work, (T*)cache, rows, n_new, R, hist, ring, start, pos_dev);
  else
    latent_append_kernel<T, false><<<(unsigned)blocks, 256, 0, stream>>>((const T*)raw, ld_raw, weight, eps, (T*)work, (T*)cache, rows, n_new, R, hist, ring, start, pos_dev);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

int launch_latent_append(const void* raw, int64_t ld_raw, const float* weight, float eps, void* work, void* cache, int64_t B, int64_t n_new, int64_t R,
                         int64_t hist, int64_t ring, int64_t start, const int* pos_dev, int dtype, cudaStream_t stream) {
  return dtype == B200_BF16 ? append_typed<__nv_bfloat16>(raw, ld_raw, weight, eps, work, cache, B, n_new, R, hist, ring, start, pos_dev, stream)
                            : append_typed<float>(raw, ld_raw, weight, eps, work, cache, B, n_new, R, hist, ring, start, pos_dev, stream);
}

int launch_latent_gather(const void* cache, void* work, int64_t B, int64_t n_new, int64_t R, int64_t hist, int64_t ring, int64_t start, int dtype,
                         cudaStream_t stream) {
  const int64_t rows = B * hist, blocks = (rows + 7) / 8;
  if (blocks > 0x7fffffffLL) return B200_ERR_BAD_ARGUMENT;
  if (dtype == B200_BF16)
    latent_gather_kernel<__nv_bfloat16><<<(unsigned)blocks, 256, 0, stream>>>((const __nv_bfloat16*)cache, (__nv_bfloat16*)work, rows, n_new, R, hist, ring, start);
  else
    latent_gather_kernel<float><<<(unsigned)blocks, 256, 0, stream>>>((const float*)cache, (float*)work, rows, n_new, R, hist, ring, start);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

int launch_window_attention(const void* q, int64_t ld_q, const void* k, int64_t ld_k, const void* v, int64_t ld_v, void* out, int64_t ld_out,
                            int64_t B, int64_t n_new, int64_t hist, int64_t heads, int64_t dim, int64_t vdim, int64_t window, float scale,
                            const float* sink, int dtype, int* status_word, cudaStream_t stream) {
  {
    const int st = launch_window_attention_sm100(q, ld_q, k, ld_k, v, ld_v, out, ld_out, B, n_new, hist, heads, dim, vdim, window, scale, sink, dtype,
                                                 status_word, stream);
    if (st != B200_ERR_UNSUPPORTED) return st;
  }
  if (dtype == B200_BF16)
    return window_typed<__nv_bfloat16>(q, ld_q, k, ld_k, v, ld_v, out, ld_out, B, n_new, hist, heads, dim, vdim, window, scale, sink, stream);
  return window_typed<float>(q, ld_q, k, ld_k, v, ld_v, out, ld_out, B, n_new, hist, heads, dim, vdim, window, scale, sink, stream);
}

size_t latent_decode_workspace_bytes(int64_t B, int64_t heads, int64_t R, int64_t window, int dtype) {
  const size_t simple = (size_t)(2 * B * heads * R) * 4;
  if (dtype != B200_BF16) return simple;
  const size_t mma = latent_decode_mma_workspace_bytes(B, heads, R, window);
  return mma > simple ? mma : simple;
}

int launch_latent_decode(const void* q, int64_t ld_q, const void* w_uk, const void* w_uv, const void* cache, void* out, int64_t ld_out, int64_t B,
                         int64_t heads, int64_t dim, int64_t vdim, int64_t R, int64_t ring, int64_t window, float scale, const float* sink,
                         int dtype, const int* pos_dev, void* workspace, cudaStream_t stream) {
  if (B * heads > 0x7fffffffLL || heads > 65535 || B > 65535 * kBatchTile) return B200_ERR_BAD_ARGUMENT;
  if (dtype == B200_BF16) {
    const int st = launch_latent_decode_mma(q, ld_q, w_uk, w_uv, cache, out, ld_out, B, heads, dim, vdim, R, ring, window, scale, sink, pos_dev, workspace, stream);
    if (st != B200_ERR_UNSUPPORTED) return st;
  }
  if (dtype == B200_BF16)
    return decode_typed<__nv_bfloat16>(q, ld_q, w_uk, w_uv, cache, out, ld_out, B, heads, dim, vdim, R, ring, window, scale, sink, pos_dev, workspace, stream);
  return decode_typed<float>(q, ld_q, w_uk, w_uv, cache, out, ld_out, B, heads, dim, vdim, R, ring, window, scale, sink, pos_dev, workspace, stream);
}

}  // namespace b200
