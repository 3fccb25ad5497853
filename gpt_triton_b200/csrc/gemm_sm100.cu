// Entry points of the tcgen05 GEMM (gemm_sm100.cuh): plain, with row statistics, and LayerNorm-aware, and the small
// kernels that merge the per-slice partial results its epilogues leave.
#include "gemm_sm100.cuh"

namespace b200 {

// Row argmax (and optionally the row log-sum-exp) from the per-slice partials the GEMM epilogue wrote.  A block
// covers 32 rows with 8 threads per row: thread (x, y) walks slices y, y + 8, ... of row x (32 consecutive rows of
// one slice are one 128-byte line), then the 8 partial results of a row are merged through shared memory.  Strict
// '>' within a thread and the lower column on equal values across threads keep the lowest column among equal maxima.
// A partial's column is either exact (>= 0) or -(c0 + 1): "somewhere in the 32 stored columns starting at c0"; for the
// row's winner that chunk of the stored product is read back and its first column equal to the maximum taken.
constexpr int kReduceRows = 32, kReduceSplit = 8;
__device__ __forceinline__ int partial_column(int enc) { return enc < 0 ? -enc - 1 : enc; }
__global__ void __launch_bounds__(kReduceRows * kReduceSplit)
argmax_reduce_kernel(const float* __restrict__ val, const int* __restrict__ idx, const float* __restrict__ sum, int64_t ld, int slices,
                     int64_t M, int64_t* __restrict__ out, float* __restrict__ lse_out, const void* __restrict__ product, int64_t ld_product,
                     int product_is_bf16, int64_t N) {
  __shared__ float s_val[kReduceSplit][kReduceRows];
  __shared__ int s_idx[kReduceSplit][kReduceRows];
  __shared__ float s_sum[kReduceSplit][kReduceRows];
  const int x = threadIdx.x & (kReduceRows - 1), y = threadIdx.x / kReduceRows;
  const int64_t row = (int64_t)blockIdx.x * kReduceRows + x;
  pdl_launch_dependents();
  pdl_wait();
  float best = -INFINITY, total = 0.f;
  int where = 0x7fffffff;
  if (row < M) {
    for (int s = y; s < slices; s += kReduceSplit) {
      const float v = val[(int64_t)s * ld + row];
      if (v > best) {
        if (sum) total *= __expf(best - v);  // re-base what was summed so far (0 * exp(-inf) = 0 the first time)
        best = v, where = idx[(int64_t)s * ld + row];
      }
      if (sum && v > -INFINITY) total += sum[(int64_t)s * ld + row] * __expf(v - best);
    }
  }
  s_val[y][x] = best, s_idx[y][x] = where, s_sum[y][x] = total;
  __syncthreads();
  if (y == 0 && row < M) {
#pragma unroll
    for (int k = 1; k < kReduceSplit; ++k) {
      const float v = s_val[k][x];
      const int w = s_idx[k][x];
      const float t = s_sum[k][x];
      if (v > best || (v == best && w != 0x7fffffff && (where == 0x7fffffff || partial_column(w) < partial_column(where)))) {
        total = total * (best > -INFINITY ? __expf(best - v) : 0.f) + t;
        best = v, where = w;
      } else if (v > -INFINITY) {
        total += t * __expf(v - best);
      }
    }
    if (where == 0x7fffffff) {
      where = 0;
    } else if (where < 0) {
      const int c0 = -where - 1;
      where = c0;
      if (product) {
        for (int i = 0; i < 32 && c0 + i < N; ++i) {
          const float pv = product_is_bf16 ? to_float(static_cast<const __nv_bfloat16*>(product)[row * ld_product + c0 + i])
                                           : to_float(static_cast<const __half*>(product)[row * ld_product + c0 + i]);
          if (pv == best) {
            where = c0 + i;
            break;
          }
        }
      }
    }
    out[row] = where;
    if (lse_out) lse_out[row] = best + logf(total);
  }
}

static int launch_argmax_reduce(const float* val, const int* idx, const float* sum, int64_t ld, int slices, int64_t M, int64_t* out, float* lse_out,
                                const void* product, int64_t ld_product, int product_dtype, int64_t N, cudaStream_t stream) {
  LaunchSetup ls(dim3((unsigned)((M + kReduceRows - 1) / kReduceRows)), dim3(kReduceRows * kReduceSplit), 0, stream);
  const int is_bf16 = product_dtype == B200_BF16;
  if (product_dtype == B200_F32) product = nullptr;  // fp32 products never defer the column
  const cudaError_t e = cudaLaunchKernelEx(&ls.cfg, argmax_reduce_kernel, val, idx, sum, ld, slices, M, out, lse_out, product, ld_product, is_bf16, N);
  note_launches(1);
  return status_from_cuda(e);
}

// Merges the per-slice (mean, centred sum of squares) pairs a LN == 2 epilogue wrote into one (mean, rstd) per row:
// mean = sum_s n_s mean_s / n,  M2 = sum_s M2_s + sum_s n_s (mean_s - mean)^2  (every term non-negative: no
// cancellation),  rstd = 1 / sqrt(M2 / n + eps); also writes the row's extension for a consuming GEMM.  One thread per
// row; the slices of 32 consecutive rows are consecutive in memory.
template <typename T>
__global__ void __launch_bounds__(256)
ln_stats_from_moments_kernel(const float2* __restrict__ moments, int64_t ld, int slices, int slice_cols, int cols, float eps, int64_t M,
                             float2* __restrict__ stats, T* __restrict__ ext) {
  const int64_t row = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  const bool active = row < M;  // (no early return: the whole warp takes part in the shuffles below)
  const int64_t rrow = active ? row : M - 1;
  float wsum = 0.f;
  for (int s = 0; s < slices; ++s) wsum = fmaf((float)min(slice_cols, cols - s * slice_cols), moments[(int64_t)s * ld + rrow].x, wsum);
  const float mean = wsum / (float)cols;
  float m2 = 0.f;
  for (int s = 0; s < slices; ++s) {
    const float2 part = moments[(int64_t)s * ld + rrow];
    const float d = part.x - mean;
    m2 += fmaf((float)min(slice_cols, cols - s * slice_cols) * d, d, part.y);
  }
  const float sd = sqrtf(m2 / (float)cols + eps);
  if (active) stats[row] = make_float2(mean, 1.0f / sd);
  if (ext) {
    // The extensions of a warp's 32 consecutive rows are 4 KB of consecutive memory (16 meaningful bytes and 112
    // zero bytes per row): written as 8 fully coalesced 512-byte warp stores, the heads fetched by shuffle.
    const uint4 head = ln_ext_head<T>(mean, sd);
    const int lane = threadIdx.x & 31;
    const int64_t warp_row0 = row - lane;
    uint4* dst = reinterpret_cast<uint4*>(ext + warp_row0 * kLnExtCols);
    constexpr int kChunksPerRow = kLnExtCols * 2 / 16;  // 8
#pragma unroll
    for (int i = 0; i < kChunksPerRow; ++i) {
      const int chunk = i * 32 + lane;          // 16-byte chunk of the warp's 4 KB
      const int src = chunk / kChunksPerRow;    // the row (lane) it belongs to
      uint4 v;
      v.x = __shfl_sync(0xffffffffu, head.x, src);
      v.y = __shfl_sync(0xffffffffu, head.y, src);
      v.z = __shfl_sync(0xffffffffu, head.z, src);
      v.w = __shfl_sync(0xffffffffu, head.w, src);
      if (chunk % kChunksPerRow != 0) v = make_uint4(0u, 0u, 0u, 0u);
      if (warp_row0 + src < M) dst[chunk] = v;
    }
  }
}

size_t gemm_ln_workspace_bytes(int64_t M, int64_t N) {
  if (M <= 0 || N <= 0) return 0;
  const int64_t slices = (N + gemm::NARROW_BN - 1) / gemm::NARROW_BN;  // (the narrow-tile kernel's slices; the wide kernel uses every other one)
  return (size_t)(slices * ((M + 63) / 64 * 64)) * 8;
}

// GEMM with a LayerNorm on either side of it (16-bit data, staged epilogue only):
//  * consumer (ln_stats != NULL): A holds raw rows x whose LayerNorm is folded into this GEMM: ln_stats[row] =
//    (mean, rstd) of x's rows and a_ext [M, kLnExtCols] their extension (both written by one of the statistics
//    producers), B holds the weights already multiplied by the LayerNorm weight and b_ext [N, kLnExtCols] their
//    extension (both written by fold_layernorm_kernel); `bias` is not used (it is inside b_ext);
//  * producer (stats_out != NULL): plain GEMM that also leaves stats_out[row] = (mean, rstd over N columns, with eps)
//    and ext_out [M, kLnExtCols] of the rows it stores, for a following consumer; `workspace`
//    (gemm_ln_workspace_bytes) holds the per-slice moments.
int launch_gemm_ln(const void* a, const void* b, const void* bias, const void* residual, void* out, int64_t M, int64_t N, int64_t K, int64_t lda,
                   int64_t ldb, int64_t ld_res, int64_t ld_out, int op_dtype, int io_dtype, int add_gelu, const float* ln_stats,
                   const void* a_ext, const void* b_ext, float* stats_out, void* ext_out, float eps, void* workspace, size_t workspace_bytes,
                   int* status_word, cudaStream_t stream) {
  using namespace gemm;
  if (M == 0 || N == 0) return B200_OK;
  if (K < 1 || M < 0 || N < 0) return B200_ERR_BAD_ARGUMENT;
  if (op_dtype != B200_F16 && op_dtype != B200_BF16) return B200_ERR_BAD_ARGUMENT;
  if (io_dtype != B200_F16 && io_dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (!a || !b || !out) return B200_ERR_BAD_ARGUMENT;
  if ((ln_stats != nullptr) == (stats_out != nullptr)) return B200_ERR_BAD_ARGUMENT;  // exactly one of the two roles per launch
  if ((reinterpret_cast<uintptr_t>(a) & 15) || (reinterpret_cast<uintptr_t>(b) & 15) || lda % 8 || ldb % 8 || lda < K || ldb < K)
    return B200_ERR_ALIGNMENT;
  if (ld_out < N || (residual && ld_res < N)) return B200_ERR_BAD_ARGUMENT;
  if (M > 0x7fffffffLL - 256 || N > 0x7fffffffLL - 256 || K > 0x7fffffffLL - 64) return B200_ERR_BAD_ARGUMENT;
  LnArgs ln;
  if (op_dtype != io_dtype) return B200_ERR_UNSUPPORTED;  // the extensions are written in the storage type and fed to the tensor cores as they are
  if (ln_stats) {
    if (!a_ext || !b_ext || (reinterpret_cast<uintptr_t>(ln_stats) & 7) || (reinterpret_cast<uintptr_t>(a_ext) & 15) ||
        (reinterpret_cast<uintptr_t>(b_ext) & 15))
      return B200_ERR_BAD_ARGUMENT;
    ln.stats = reinterpret_cast<const float2*>(ln_stats), ln.a_ext = a_ext, ln.b_ext = b_ext;
  } else {
    if (add_gelu || !ext_out || (reinterpret_cast<uintptr_t>(stats_out) & 7) || (reinterpret_cast<uintptr_t>(ext_out) & 15)) return B200_ERR_BAD_ARGUMENT;
    if (!workspace || workspace_bytes < gemm_ln_workspace_bytes(M, N) || (reinterpret_cast<uintptr_t>(workspace) & 15)) return B200_ERR_WORKSPACE;
    ln.stats_out = reinterpret_cast<float2*>(workspace), ln.stats_out_ld = (M + 63) / 64 * 64;
  }
  const ArgmaxPartials none{nullptr, nullptr, nullptr, 0};
  int st;
#define B200_GEMM_LN_DISPATCH(T)                                                                                                                 \
  st = ln_stats ? (add_gelu ? launch_typed<T, true, 0, 1>(a, b, nullptr, residual, out, M, N, K, lda, ldb, ld_res, ld_out, op_dtype, none, status_word, \
                                                          stream, nullptr, nullptr, ln)                                                          \
                            : launch_typed<T, false, 0, 1>(a, b, nullptr, residual, out, M, N, K, lda, ldb, ld_res, ld_out, op_dtype, none, status_word, \
                                                           stream, nullptr, nullptr, ln))                                                        \
                : launch_typed<T, false, 0, 2>(a, b, bias, residual, out, M, N, K, lda, ldb, ld_res, ld_out, op_dtype, none, status_word, stream, \
                                               nullptr, nullptr, ln)
  if (io_dtype == B200_F16) B200_GEMM_LN_DISPATCH(__half);
  else B200_GEMM_LN_DISPATCH(__nv_bfloat16);
#undef B200_GEMM_LN_DISPATCH
  if (st != B200_OK || !stats_out) return st;
  // width of the column slices whose moments the GEMM left: the wide kernel's epilogue warps cover EPI_COLS columns, a
  // narrow tile NARROW_BN
  const bool narrow = io_dtype == B200_F16 ? takes_narrow_tiles<__half, 0>(M, out, ld_out, residual, ld_res)
                                           : takes_narrow_tiles<__nv_bfloat16, 0>(M, out, ld_out, residual, ld_res);
  const int slice_cols = narrow ? NARROW_BN : EPI_COLS;
  const int slices = (int)((N + slice_cols - 1) / slice_cols);
  LaunchSetup ls(dim3((unsigned)((M + 255) / 256)), dim3(256), 0, stream);
  const cudaError_t e =
      io_dtype == B200_F16
          ? cudaLaunchKernelEx(&ls.cfg, ln_stats_from_moments_kernel<__half>, (const float2*)ln.stats_out, ln.stats_out_ld, slices, slice_cols,
                               (int)N, eps, M, reinterpret_cast<float2*>(stats_out), static_cast<__half*>(ext_out))
          : cudaLaunchKernelEx(&ls.cfg, ln_stats_from_moments_kernel<__nv_bfloat16>, (const float2*)ln.stats_out, ln.stats_out_ld, slices,
                               slice_cols, (int)N, eps, M, reinterpret_cast<float2*>(stats_out), static_cast<__nv_bfloat16*>(ext_out));
  note_launches(1);
  return status_from_cuda(e);
}

int launch_gemm(const void* a, const void* b, const void* bias, const void* residual, void* out, int64_t M, int64_t N,
                int64_t K, int64_t lda, int64_t ldb, int64_t ld_res, int64_t ld_out, int op_dtype, int io_dtype,
                int add_gelu, int* status_word, cudaStream_t stream) {
  return launch_gemm_argmax(a, b, bias, residual, out, M, N, K, lda, ldb, ld_res, ld_out, op_dtype, io_dtype, add_gelu, nullptr, nullptr,
                            nullptr, 0, status_word, stream);
}

size_t gemm_argmax_workspace_bytes(int64_t M, int64_t N) {
  if (M <= 0 || N <= 0) return 0;
  const int64_t slices = (N + gemm::BN - 1) / gemm::BN * (gemm::BN / gemm::EPI_COLS);
  const int64_t ld = (M + 63) / 64 * 64;
  return (size_t)(slices * ld) * 12;  // maximum, column, sum of exponentials
}

int launch_gemm_argmax(const void* a, const void* b, const void* bias, const void* residual, void* out, int64_t M, int64_t N,
                       int64_t K, int64_t lda, int64_t ldb, int64_t ld_res, int64_t ld_out, int op_dtype, int io_dtype,
                       int add_gelu, int64_t* argmax_out, float* lse_out, void* workspace, size_t workspace_bytes, int* status_word,
                       cudaStream_t stream) {
  using namespace gemm;
  ArgmaxPartials am{nullptr, nullptr, nullptr, 0};
  if (argmax_out) {
    const size_t need = gemm_argmax_workspace_bytes(M, N);
    if (need > 0 && (!workspace || workspace_bytes < need || (reinterpret_cast<uintptr_t>(workspace) & 15))) return B200_ERR_WORKSPACE;
    am.ld = (M + 63) / 64 * 64;
    const int64_t slices = (N + BN - 1) / BN * (BN / EPI_COLS);
    am.val = static_cast<float*>(workspace);
    am.idx = reinterpret_cast<int*>(am.val + slices * am.ld);
    if (lse_out) am.sum = am.val + 2 * slices * am.ld;
  }
  if (M == 0 || N == 0) return B200_OK;
  if (K < 1 || M < 0 || N < 0) return B200_ERR_BAD_ARGUMENT;
  if (op_dtype != B200_F16 && op_dtype != B200_BF16) return B200_ERR_BAD_ARGUMENT;
  if (!a || !b || !out) return B200_ERR_BAD_ARGUMENT;
  if ((reinterpret_cast<uintptr_t>(a) & 15) || (reinterpret_cast<uintptr_t>(b) & 15) || lda % 8 || ldb % 8 || lda < K || ldb < K)
    return B200_ERR_ALIGNMENT;
  if (ld_out < N || (residual && ld_res < N)) return B200_ERR_BAD_ARGUMENT;
  if (M > 0x7fffffffLL - 256 || N > 0x7fffffffLL - 256 || K > 0x7fffffffLL - 64) return B200_ERR_BAD_ARGUMENT;
  if (argmax_out && add_gelu) return B200_ERR_UNSUPPORTED;  // row statistics are built for the plain and residual epilogues only
  int st = B200_ERR_BAD_ARGUMENT;
#define B200_GEMM_DISPATCH(T)                                                                                                              \
  st = (argmax_out && lse_out) ? launch_typed<T, false, 2>(a, b, bias, residual, out, M, N, K, lda, ldb, ld_res, ld_out, op_dtype, am, status_word, stream) \
       : argmax_out ? launch_typed<T, false, 1>(a, b, bias, residual, out, M, N, K, lda, ldb, ld_res, ld_out, op_dtype, am, status_word, stream)  \
       : add_gelu ? launch_typed<T, true, 0>(a, b, bias, residual, out, M, N, K, lda, ldb, ld_res, ld_out, op_dtype, am, status_word, stream)  \
                  : launch_typed<T, false, 0>(a, b, bias, residual, out, M, N, K, lda, ldb, ld_res, ld_out, op_dtype, am, status_word, stream)
  switch (io_dtype) {
    case B200_F32: B200_GEMM_DISPATCH(float); break;
    case B200_F16: B200_GEMM_DISPATCH(__half); break;
    case B200_BF16: B200_GEMM_DISPATCH(__nv_bfloat16); break;
  }
#undef B200_GEMM_DISPATCH
  if (st != B200_OK || !argmax_out) return st;
  const int64_t slices = (N + BN - 1) / BN * (BN / EPI_COLS);
  return launch_argmax_reduce(am.val, am.idx, am.sum, am.ld, (int)slices, M, argmax_out, lse_out, out, ld_out, io_dtype, N, stream);
}

// Row statistics of A B^T (+ bias) without storing the product: argmax, log-sum-exp and, optionally, the value at a
// per-row target column, all taken from the values as they would be rounded to `round_dtype` (fp16 or bf16).
int launch_gemm_rowstats(const void* a, const void* b, const void* bias, int64_t M, int64_t N, int64_t K, int64_t lda, int64_t ldb,
                         int op_dtype, int round_dtype, const int64_t* targets, int64_t* argmax_out, float* lse_out, float* target_out,
                         void* workspace, size_t workspace_bytes, int* status_word, cudaStream_t stream) {
  using namespace gemm;
  if (!argmax_out || (targets != nullptr) != (target_out != nullptr)) return B200_ERR_BAD_ARGUMENT;
  if (K < 1 || M < 0 || N < 0) return B200_ERR_BAD_ARGUMENT;
  if (M == 0 || N == 0) return B200_OK;
  if (op_dtype != B200_F16 && op_dtype != B200_BF16) return B200_ERR_BAD_ARGUMENT;
  if (round_dtype != B200_F16 && round_dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (!a || !b) return B200_ERR_BAD_ARGUMENT;
  if ((reinterpret_cast<uintptr_t>(a) & 15) || (reinterpret_cast<uintptr_t>(b) & 15) || lda % 8 || ldb % 8 || lda < K || ldb < K)
    return B200_ERR_ALIGNMENT;
  if (M > 0x7fffffffLL - 256 || N > 0x7fffffffLL - 256 || K > 0x7fffffffLL - 64) return B200_ERR_BAD_ARGUMENT;
  const size_t need = gemm_argmax_workspace_bytes(M, N);
  if (!workspace || workspace_bytes < need || (reinterpret_cast<uintptr_t>(workspace) & 15)) return B200_ERR_WORKSPACE;
  ArgmaxPartials am;
  am.ld = (M + 63) / 64 * 64;
  const int64_t slices = (N + BN - 1) / BN * (BN / EPI_COLS);
  am.val = static_cast<float*>(workspace);
  am.idx = reinterpret_cast<int*>(am.val + slices * am.ld);
  am.sum = lse_out ? am.val + 2 * slices * am.ld : nullptr;
  int st;
  if (round_dtype == B200_F16)
    st = launch_typed<__half, false, 3>(a, b, bias, nullptr, nullptr, M, N, K, lda, ldb, 0, N, op_dtype, am, status_word, stream, targets, target_out);
  else
    st = launch_typed<__nv_bfloat16, false, 3>(a, b, bias, nullptr, nullptr, M, N, K, lda, ldb, 0, N, op_dtype, am, status_word, stream, targets, target_out);
  if (st != B200_OK) return st;
  return launch_argmax_reduce(am.val, am.idx, am.sum, am.ld, (int)slices, M, argmax_out, lse_out, nullptr, 0, round_dtype, N, stream);
}

}  // namespace b200
