// Differential attention: per head two softmax maps over the same values, subtracted, normed and gated; sliding window,
// grouped key/value heads, soft-capped scores.  Prompts run pair_attention_sm100.cu and single tokens pair_decode.cu where they
// fit; the kernel of this file takes any sizes, both storage types, prompts and
// single tokens; fp32 storage is computed in true 32-bit throughout.
#include "common.cuh"

namespace b200 {
namespace {

// One warp per (query, head): 32 keys at a time, one per lane, online softmax for both maps; the two output rows live in
// shared memory (a lane owns every 32nd column, so nothing needs a barrier).
constexpr int kQueryWarps = 4;
template <typename T, typename TV>
__global__ void __launch_bounds__(32 * kQueryWarps)
pair_attention_kernel(b200_pair_attention_args p, int64_t n_items) {
  extern __shared__ float smem_f[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int dim = (int)p.dim, vdim = (int)p.vdim;
  float* qs = smem_f + warp * 2 * (dim + vdim);
  float* o = qs + 2 * dim;
  const int64_t item = (int64_t)blockIdx.x * kQueryWarps + warp;
  if (item >= n_items) return;
  const int64_t h = item % p.heads, row = item / p.heads, b = row / p.n, t = row % p.n;
  const int64_t g = h / (p.heads / p.kv_heads);
  const T* q = static_cast<const T*>(p.q) + row * p.ld_q + h * 2 * dim;
  for (int c = lane; c < 2 * dim; c += 32) qs[c] = to_float(q[c]);
  for (int c = lane; c < 2 * vdim; c += 32) o[c] = 0.f;
  __syncwarp();
  // positions of the keys: those of the work rows, or those of the ring
  const int64_t last = p.pos_dev ? (int64_t)p.pos_dev[0] : p.hist + t, first = last + 1 > p.window ? last + 1 - p.window : 0;
  const T* kb = static_cast<const T*>(p.k) + b * p.k_batch + g * p.k_head;
  const TV* vb = static_cast<const TV*>(p.v) + b * p.v_batch + g * p.v_head;
  const float inv_cap = p.softcap > 0.f ? 1.0f / p.softcap : 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  for (int64_t j0 = first; j0 <= last; j0 += 32) {
    const int64_t j = j0 + lane;
    const int64_t slot = p.ring > 0 ? j % p.ring : j;
    float w[2], mult[2];
#pragma unroll
    for (int map = 0; map < 2; ++map) {
      float s = -INFINITY;
      if (j <= last) {
        const T* kr = kb + slot * p.k_row + map * dim;
        float a = 0.f;
        for (int c = 0; c < dim; ++c) a = fmaf(qs[map * dim + c], to_float(kr[c]), a);
        s = a * p.scale;
        if (p.softcap > 0.f) s = p.softcap * tanhf(s * inv_cap);
      }
      float mb = s;
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) mb = fmaxf(mb, __shfl_xor_sync(0xffffffffu, mb, off));
      const float m_new = fmaxf(m[map], mb);
      mult[map] = expf(m[map] - m_new);
      w[map] = expf(s - m_new);
      l[map] = l[map] * mult[map] + warp_sum(w[map]);
      m[map] = m_new;
    }
    const int n = (int)(last - j0 + 1 < 32 ? last - j0 + 1 : 32);
    for (int c0 = 0; c0 < vdim; c0 += 32) {
      const int c = c0 + lane;
      float a0 = c < vdim ? o[c] * mult[0] : 0.f, a1 = c < vdim ? o[vdim + c] * mult[1] : 0.f;
      for (int i = 0; i < n; ++i) {
        const float w0 = __shfl_sync(0xffffffffu, w[0], i), w1 = __shfl_sync(0xffffffffu, w[1], i);
        const int64_t si = __shfl_sync(0xffffffffu, slot, i);
        if (c < vdim) {
          const float f = to_float(vb[si * p.v_row + c]);
          a0 = fmaf(w0, f, a0), a1 = fmaf(w1, f, a1);
        }
      }
      if (c < vdim) o[c] = a0, o[vdim + c] = a1;
    }
  }
  const float lambda = p.lambda[0], r0 = 1.0f / l[0], r1 = 1.0f / l[1];
  float sq = 0.f;
  for (int c = lane; c < vdim; c += 32) {
    const float d = o[c] * r0 - lambda * (o[vdim + c] * r1);
    o[c] = d;
    sq = fmaf(d, d, sq);
  }
  const float f = p.out_scale / sqrtf(warp_sum(sq) / (float)vdim + p.eps) * to_float(static_cast<const T*>(p.gate)[row * p.ld_gate + h]);
  T* out = static_cast<T*>(p.out) + row * p.ld_out + h * vdim;
  for (int c = lane; c < vdim; c += 32) out[c] = from_float<T>(o[c] * f);
}

template <typename T, typename TV>
int launch_any(const b200_pair_attention_args& p, cudaStream_t stream) {
  const int64_t n = p.B * p.n * p.heads, blocks = (n + kQueryWarps - 1) / kQueryWarps;
  const size_t smem = (size_t)kQueryWarps * 2 * (p.dim + p.vdim) * 4;
  if (smem > 48 * 1024 || blocks > 0x7fffffffLL) return B200_ERR_UNSUPPORTED;
  pair_attention_kernel<T, TV><<<(unsigned)blocks, 32 * kQueryWarps, smem, stream>>>(p, n);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

}  // namespace

int pair_attention_v_dtype(int64_t dim, int64_t vdim, int dtype) {
  return pair_attention_sm100_takes(dim, vdim, dtype) ? B200_F16 : dtype;
}

int64_t pair_attention_workspace_bytes(const b200_pair_attention_args& p) {
  (void)p;
  return 0;
}

int launch_pair_attention(const b200_pair_attention_args& p, cudaStream_t stream) {
  const int st = p.pos_dev ? launch_pair_decode(p, stream) : launch_pair_attention_sm100(p, stream);
  if (st != B200_ERR_UNSUPPORTED) return st;
  if (p.dtype == B200_F32) return launch_any<float, float>(p, stream);
  if (p.v_dtype == B200_F16) return launch_any<__nv_bfloat16, __half>(p, stream);
  return launch_any<__nv_bfloat16, __nv_bfloat16>(p, stream);
}

}  // namespace b200
