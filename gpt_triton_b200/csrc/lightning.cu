// Decayed linear attention: per head S <- decay * S + k v^T, o = S^T q with an fp32 state, over one token or many.
//
// recurrent kernel: token by token, exactly the recurrence, any sizes, both storage types.  A block owns 32 columns of
// one head's state in registers (four warps split the rows); tokens are staged 16 at a time in shared memory.
#include "common.cuh"

namespace b200 {
namespace {

constexpr int kCols = 32, kRowWarps = 4, kTokens = 16;

template <typename T, int RPW>  // RPW: state rows per warp
__global__ void __launch_bounds__(32 * kRowWarps)
recurrent_kernel(const T* __restrict__ qkvg, int64_t ld, int64_t off_k, int64_t off_v, int64_t off_g, const double* __restrict__ decay,
                 const float* __restrict__ weight, float* __restrict__ state, int fresh, T* __restrict__ y, int64_t ld_y, float* __restrict__ sumsq,
                 int64_t ld_sumsq, int n_tok, int heads, int dim, int vdim) {
  __shared__ __align__(16) float qs[kTokens][RPW * kRowWarps], ks[kTokens][RPW * kRowWarps];
  __shared__ float vs[kTokens][kCols];
  __shared__ float part[kTokens][kRowWarps][kCols];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int vblocks = (vdim + kCols - 1) / kCols;
  const int vb = blockIdx.x % vblocks;
  const int h = (blockIdx.x / vblocks) % heads;
  const int64_t b = blockIdx.x / (vblocks * heads);
  const int col = vb * kCols + lane;
  const bool col_ok = col < vdim;
  const int row0 = warp * RPW;
  float* st = state + ((b * heads + h) * dim) * (int64_t)vdim + col;
  const float lam = (float)decay[h];
  float s[RPW];
#pragma unroll
  for (int i = 0; i < RPW; ++i) s[i] = (!fresh && col_ok && row0 + i < dim) ? st[(int64_t)(row0 + i) * vdim] : 0.f;
  for (int t0 = 0; t0 < n_tok; t0 += kTokens) {
    const int n = min(kTokens, n_tok - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < kTokens * RPW * kRowWarps; i += 32 * kRowWarps) {
      const int t = i / (RPW * kRowWarps), d = i % (RPW * kRowWarps);
      float qv = 0.f, kv = 0.f;
      if (t < n && d < dim) {
        const T* row = qkvg + (b * n_tok + t0 + t) * ld + h * dim + d;
        qv = to_float(row[0]), kv = to_float(row[off_k]);
      }
      qs[t][d] = qv, ks[t][d] = kv;
    }
    for (int t = warp; t < n; t += kRowWarps) vs[t][lane] = col_ok ? to_float(qkvg[(b * n_tok + t0 + t) * ld + off_v + h * vdim + col]) : 0.f;
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float v = vs[t][lane];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < RPW; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(&ks[t][row0 + i]);
        const float4 q4 = *reinterpret_cast<const float4*>(&qs[t][row0 + i]);
        s[i] = fmaf(lam, s[i], k4.x * v), o = fmaf(s[i], q4.x, o);
        s[i + 1] = fmaf(lam, s[i + 1], k4.y * v), o = fmaf(s[i + 1], q4.y, o);
        s[i + 2] = fmaf(lam, s[i + 2], k4.z * v), o = fmaf(s[i + 2], q4.z, o);
        s[i + 3] = fmaf(lam, s[i + 3], k4.w * v), o = fmaf(s[i + 3], q4.w, o);
      }
      part[t][warp][lane] = o;
    }
    __syncthreads();
    for (int t = warp; t < n; t += kRowWarps) {
      const float o = (part[t][0][lane] + part[t][1][lane]) + (part[t][2][lane] + part[t][3][lane]);
      const int64_t row = b * n_tok + t0 + t;
      if (col_ok) {
        const int64_t c = (int64_t)h * vdim + col;
        y[row * ld_y + c] = from_float<T>(o * weight[c] * to_float(qkvg[row * ld + off_g + c]));
      }
      const float sq = warp_sum(col_ok ? o * o : 0.f);
      if (lane == 0) sumsq[(int64_t)(h * vblocks + vb) * ld_sumsq + row] = sq;
    }
  }
#pragma unroll
  for (int i = 0; i < RPW; ++i)
    if (col_ok && row0 + i < dim) st[(int64_t)(row0 + i) * vdim] = s[i];
}

struct Args {
  const void* qkvg;
  int64_t ld, off_k, off_v, off_g;
  const double* decay;
  const float* weight;
  float* state;
  int fresh;
  void* y;
  int64_t ld_y;
  float* sumsq;
  int64_t ld_sumsq, B, n_tok, heads, dim, vdim;
};

template <typename T>
int launch_recurrent(const Args& a, cudaStream_t stream) {
  const int64_t blocks = a.B * a.heads * ((a.vdim + kCols - 1) / kCols);
  if (blocks > 0x7fffffffLL || a.n_tok > 0x7fffffffLL) return B200_ERR_BAD_ARGUMENT;
#define B200_RECURRENT(RPW)                                                                                                                   \
  recurrent_kernel<T, RPW><<<(unsigned)blocks, 32 * kRowWarps, 0, stream>>>((const T*)a.qkvg, a.ld, a.off_k, a.off_v, a.off_g, a.decay, a.weight,   \
                                                                            a.state, a.fresh, (T*)a.y, a.ld_y, a.sumsq, a.ld_sumsq, (int)a.n_tok, \
                                                                            (int)a.heads, (int)a.dim, (int)a.vdim)
  if (a.dim <= 16) B200_RECURRENT(4);
  else if (a.dim <= 32) B200_RECURRENT(8);
  else if (a.dim <= 64) B200_RECURRENT(16);
  else if (a.dim <= 128) B200_RECURRENT(32);
  else if (a.dim <= 256) B200_RECURRENT(64);
  else return B200_ERR_UNSUPPORTED;
#undef B200_RECURRENT
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

}  // namespace

int64_t decayed_attention_slices(int64_t n_tok, int64_t heads, int64_t dim, int64_t vdim, int dtype) {
  (void)n_tok, (void)dim, (void)dtype;
  return heads * ((vdim + kCols - 1) / kCols);
}

size_t decayed_attention_workspace_bytes(int64_t B, int64_t n_tok, int64_t heads, int64_t dim, int64_t vdim, int dtype) {
  (void)B, (void)n_tok, (void)heads, (void)dim, (void)vdim, (void)dtype;
  return 0;
}

int launch_decayed_attention(const void* qkvg, int64_t ld, int64_t off_k, int64_t off_v, int64_t off_g, const double* decay, const float* weight,
                             float* state, int fresh, void* y, int64_t ld_y, float* sumsq, int64_t ld_sumsq, int64_t B, int64_t n_tok, int64_t heads,
                             int64_t dim, int64_t vdim, int dtype, void* workspace, int* status_word, cudaStream_t stream) {
  (void)workspace, (void)status_word;
  const Args a{qkvg, ld, off_k, off_v, off_g, decay, weight, state, fresh, y, ld_y, sumsq, ld_sumsq, B, n_tok, heads, dim, vdim};
  return dtype == B200_BF16 ? launch_recurrent<__nv_bfloat16>(a, stream) : launch_recurrent<float>(a, stream);
}

}  // namespace b200
