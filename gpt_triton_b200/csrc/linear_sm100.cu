// 16-bit instantiations of the tcgen05 GEMM behind b200_linear: products over rows whose RMS norm is deferred to the
// epilogue (gemm_sm100.cuh, LN == 3 and 4), and the gated pairs of a feed-forward (LN == 5).
#include "gemm_sm100.cuh"

namespace b200 {
namespace {

template <typename OutT, int LN>
int launch(const b200_linear_args& p, const gemm::EpilogueArgs<OutT>& epi, cudaStream_t stream) {
  const gemm::LnArgs none;
  if (p.M <= gemm::kNarrowMaxRows)
    return gemm::launch_narrow<OutT, false, LN>(p.a, p.b, epi, p.M, p.N, p.K, p.lda, p.ldb, p.op_dtype, none, p.status_word, stream);
  return gemm::launch_wide<OutT, false, 0, LN>(p.a, p.b, epi, p.M, p.N, p.K, p.lda, p.ldb, p.op_dtype, none, p.status_word, stream);
}

template <typename OutT, int LN>
int fill_and_launch(const b200_linear_args& p, cudaStream_t stream) {
  gemm::EpilogueArgs<OutT> e;
  memset(&e, 0, sizeof(e));
  e.out = static_cast<OutT*>(p.out), e.ld_out = p.ld_out;
  e.sq_in = p.row_sumsq, e.sq_in_ld = p.row_sumsq_ld, e.sq_slices = p.row_sumsq_slices, e.sq_cols = (float)p.row_sumsq_cols;
  e.eps = p.eps, e.out_scale = p.out_scale;
  e.act_lo = p.act_lo, e.act_hi = p.act_hi, e.act_split = p.act_split;
  e.act_param = p.act_param, e.fbias = p.bias;
  e.pair_cols = p.pair_cols, e.pair_limit = p.pair_limit, e.pair_alpha = p.pair_alpha;
  e.x = p.x, e.ld_x = p.ld_x, e.gain = p.gain, e.gx = static_cast<__nv_bfloat16*>(p.gx), e.ld_gx = p.ld_gx;
  e.sq_out = p.sumsq_out, e.sq_out_ld = p.sumsq_out_ld;
  return launch<OutT, LN>(p, e, stream);
}

}  // namespace

int64_t linear_sm100_slice_cols(int64_t M) { return M <= gemm::kNarrowMaxRows ? gemm::NARROW_BN : gemm::EPI_COLS; }

int launch_linear_sm100(const b200_linear_args& p, cudaStream_t stream) {
  if (p.op_dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if ((reinterpret_cast<uintptr_t>(p.a) & 15) || (reinterpret_cast<uintptr_t>(p.b) & 15) || p.lda % 8 || p.ldb % 8) return B200_ERR_ALIGNMENT;
  if (reinterpret_cast<uintptr_t>(p.bias) & 15) return B200_ERR_ALIGNMENT;
  if (p.x) return fill_and_launch<float, 4>(p, stream);
  if (p.pair_cols) return p.out_dtype == B200_BF16 ? fill_and_launch<__nv_bfloat16, 5>(p, stream) : B200_ERR_UNSUPPORTED;
  if (p.out_dtype == B200_BF16) return fill_and_launch<__nv_bfloat16, 3>(p, stream);
  if (p.out_dtype == B200_F32) return fill_and_launch<float, 3>(p, stream);
  return B200_ERR_UNSUPPORTED;
}

}  // namespace b200
