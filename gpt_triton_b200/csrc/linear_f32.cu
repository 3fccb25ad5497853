// b200_linear in true 32-bit arithmetic: fp32 operands, fp32 multiply-adds on the CUDA cores (the tensor cores round
// fp32 operands to 10 mantissa bits), the same epilogue as the tcgen05 version.  One 64 x 64 tile per block, 16-wide
// k-steps staged in shared memory, a 4 x 4 piece per thread; any sizes and pitches.
#include "common.cuh"

namespace b200 {
namespace {

constexpr int TM = 64, TN = 64, TK = 16, PAD = 4;

__device__ __forceinline__ float activate_exact(float v, int act, float param) {
  switch (act) {
    case B200_ACT_SILU: return v / (1.0f + expf(-v));
    case B200_ACT_SIGMOID: return 1.0f / (1.0f + expf(-v));
    case B200_ACT_GELU_TANH: return 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    case B200_ACT_SOFTCAP: return param * tanhf(v / param);
  }
  return v;
}

__global__ void __launch_bounds__(256) linear_f32_kernel(b200_linear_args p) {
  __shared__ float sa[TK][TM + PAD], sb[TK][TN + PAD];
  __shared__ float srow[TM];
  const float* a = static_cast<const float*>(p.a);
  const float* b = static_cast<const float*>(p.b);
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int64_t m0 = (int64_t)blockIdx.y * TM, n0 = (int64_t)blockIdx.x * TN;
  float acc[4][4] = {};
  for (int64_t k0 = 0; k0 < p.K; k0 += TK) {
#pragma unroll
    for (int i = 0; i < TM * TK / 256; ++i) {
      const int e = tid + i * 256, r = e / TK, k = e % TK;
      const bool kin = k0 + k < p.K;
      sa[k][r] = (kin && m0 + r < p.M) ? a[(m0 + r) * p.lda + k0 + k] : 0.f;
      sb[k][r] = (kin && n0 + r < p.N) ? b[(n0 + r) * p.ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&sa[k][ty * 4]);
      const float4 bv = *reinterpret_cast<const float4*>(&sb[k][tx * 4]);
      const float ar[4] = {av.x, av.y, av.z, av.w}, br[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(ar[i], br[j], acc[i][j]);
    }
    __syncthreads();
  }
  if (tid < TM && m0 + tid < p.M) {
    float scale = p.out_scale;
    if (p.row_sumsq) {
      float s = 0.f;
      for (int i = 0; i < p.row_sumsq_slices; ++i) s += p.row_sumsq[(int64_t)i * p.row_sumsq_ld + m0 + tid];
      scale /= sqrtf(s / (float)p.row_sumsq_cols + p.eps);
    }
    srow[tid] = scale;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int64_t row = m0 + ty * 4 + i;
    const bool row_ok = row < p.M;
    const float scale = row_ok ? srow[ty * 4 + i] : 0.f;
    float sq = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int64_t col = n0 + tx * 4 + j;
      if (!row_ok || col >= p.N) continue;
      float v = acc[i][j] * scale;
      if (p.x) {
        v += p.x[row * p.ld_x + col];
        p.x[row * p.ld_x + col] = v;
        sq = fmaf(v, v, sq);
        if (p.gain) static_cast<float*>(p.gx)[row * p.ld_gx + col] = v * p.gain[col];
      } else {
        static_cast<float*>(p.out)[row * p.ld_out + col] =
            activate_exact(p.bias ? v + p.bias[col] : v, col < p.act_split ? p.act_lo : p.act_hi, p.act_param);
      }
    }
    if (p.x && p.gain) {  // (block-uniform) the 16 threads of a row are consecutive lanes
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
      if (tx == 0 && row_ok) p.sumsq_out[(int64_t)blockIdx.x * p.sumsq_out_ld + row] = sq;
    }
  }
}

}  // namespace

int64_t linear_f32_slice_cols() { return TN; }

int launch_linear_f32(const b200_linear_args& p, cudaStream_t stream) {
  if ((!p.x && p.out_dtype != B200_F32) || p.pair_cols) return B200_ERR_UNSUPPORTED;
  const int64_t nb = (p.N + TN - 1) / TN, mb = (p.M + TM - 1) / TM;
  if (mb > 65535) return B200_ERR_BAD_ARGUMENT;
  linear_f32_kernel<<<dim3((unsigned)nb, (unsigned)mb), 256, 0, stream>>>(p);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

}  // namespace b200
