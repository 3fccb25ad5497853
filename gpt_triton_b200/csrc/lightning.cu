// Decayed linear attention: per head S <- decay * S + k v^T, o = S^T q with an fp32 state, over one token or many.
//
// recurrent kernel: token by token, exactly the recurrence, any sizes, both storage types.  A block owns 32 columns of
// one head's state in registers (four warps split the rows); tokens are staged a few at a time in shared memory.
//
// chunked kernel (bf16, many tokens): 64 tokens at a time on the tensor cores.  With the state S before a chunk and
// i, j = 0..63 inside it,
//     o_i = decay^(i+1) q_i S + sum_{j<=i} decay^(i-j) (q_i . k_j) v_j
//     S  <- decay^n S + sum_j decay^(n-1-j) k_j v_j^T
// where every power has a non-negative exponent (no overflow for any decay).  q, k and v are bf16 and enter the MMAs as
// they are; whatever is fp32 by definition (the state, the decayed scores, the decayed keys) enters as the sum of two bf16
// parts, which carries 16 mantissa bits, and is accumulated and kept in fp32.  A block owns 64 columns of one head's state.
// Few sequences: the tokens are cut into segments that run side by side; a first pass computes what each segment adds to
// the state, a scan turns that into the segments' start states.
#include <atomic>

#include "mma_sync.cuh"

namespace b200 {
namespace {

using namespace warp_mma;

constexpr int kCols = 32, kRowWarps = 4;

template <typename T, int RPW>  // RPW: state rows per warp
__global__ void __launch_bounds__(32 * kRowWarps, RPW <= 32 ? 5 : 1)
recurrent_kernel(const T* __restrict__ qkvg, int64_t ld, int64_t off_k, int64_t off_v, int64_t off_g, const double* __restrict__ decay,
                 const float* __restrict__ weight, float* __restrict__ state, int fresh, T* __restrict__ y, int64_t ld_y, float* __restrict__ sumsq,
                 int64_t ld_sumsq, int n_tok, int heads, int dim, int vdim) {
  constexpr int kTokens = RPW <= 64 ? 16 : 4;  // tokens staged at a time
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
  else if (a.dim <= 512) B200_RECURRENT(128);
  else return B200_ERR_UNSUPPORTED;
#undef B200_RECURRENT
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

// ------------------------------------------------------------------ chunked kernel
constexpr int kChunk = 64, kVCols = 64, kChunkThreads = 128;

template <int DIM>
struct ChunkSmem {
  static constexpr int QK_BYTES = kChunk * DIM * 2;     // q or k tile, rows of DIM bf16
  static constexpr int V_BYTES = kChunk * kVCols * 2;
  static constexpr int STAGE_BYTES = 2 * QK_BYTES + V_BYTES;
  static constexpr int S_BYTES = DIM * kVCols * 2;      // one bf16 part of the state
  static constexpr int BYTES = 2 * STAGE_BYTES + 2 * S_BYTES;
};

// OUTPUT: the full computation.  Otherwise only the state a segment adds (starting from zero) is computed.
// blockIdx.x = (sequence, head, column block), blockIdx.y = segment of seg_len tokens (a multiple of the chunk).
template <int DIM, bool OUTPUT>
__global__ void __launch_bounds__(kChunkThreads, 2)
chunked_kernel(const __nv_bfloat16* __restrict__ qkvg, int64_t ld, int64_t off_k, int64_t off_v, int64_t off_g, const double* __restrict__ decay,
               const float* __restrict__ weight, const float* state_in, int64_t state_in_seg, float* state_out, int64_t state_out_seg, int fresh,
               __nv_bfloat16* __restrict__ y, int64_t ld_y, float* __restrict__ sumsq, int64_t ld_sumsq, int n_tok, int seg_len, int heads, int dim,
               int vdim) {
  using M = ChunkSmem<DIM>;
  constexpr int MT = DIM / 64;  // 16-row state tiles per warp
  constexpr int QROW = DIM * 2, VROW = kVCols * 2;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float pw[kChunk + 1];  // powers of the decay
  __shared__ float ws[kVCols];      // norm weights of this block's columns
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
  const int vblocks = (vdim + kVCols - 1) / kVCols;
  const int vb = blockIdx.x % vblocks, h = (blockIdx.x / vblocks) % heads;
  const int64_t b = blockIdx.x / (vblocks * heads);
  const int c0 = vb * kVCols;
  const int seg = blockIdx.y, tok0 = seg * seg_len, tok1 = min(n_tok, tok0 + seg_len);
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem);
  const uint32_t s_hi = base + 2 * M::STAGE_BYTES, s_lo = s_hi + M::S_BYTES;
  if (threadIdx.x < kVCols) ws[threadIdx.x] = OUTPUT && c0 + threadIdx.x < vdim ? weight[h * vdim + c0 + threadIdx.x] : 0.f;
  if (threadIdx.x <= kChunk) pw[threadIdx.x] = (float)pow(decay[h], (double)threadIdx.x);

  const __nv_bfloat16* rows = qkvg + b * n_tok * ld;
  auto load_chunk = [&](int t0, int stage) {
    const uint32_t sq = base + stage * M::STAGE_BYTES, sk = sq + M::QK_BYTES, sv = sk + M::QK_BYTES;
    for (int i = threadIdx.x; i < kChunk * (DIM / 8); i += kChunkThreads) {
      const int r = i / (DIM / 8), c = i % (DIM / 8);
      const bool ok = t0 + r < tok1 && c * 8 < dim;
      const __nv_bfloat16* src = ok ? rows + (int64_t)(t0 + r) * ld + h * dim + c * 8 : qkvg;
      if (OUTPUT) cp_async16(sq + swz<QROW>(r, c), src, ok);
      cp_async16(sk + swz<QROW>(r, c), ok ? src + off_k : qkvg, ok);
    }
    for (int i = threadIdx.x; i < kChunk * (kVCols / 8); i += kChunkThreads) {
      const int r = i / (kVCols / 8), c = i % (kVCols / 8);
      const bool ok = t0 + r < tok1 && c0 + c * 8 < vdim;
      cp_async16(sv + swz<VROW>(r, c), ok ? rows + (int64_t)(t0 + r) * ld + off_v + h * vdim + c0 + c * 8 : qkvg, ok);
    }
    cp_async_commit();
  };

  // this warp's state rows: MT tiles of 16, rows warp * 16 * MT + mt * 16 + {g8, g8 + 8}, columns nt * 8 + t4 * 2 + {0, 1}
  float st[MT][8][4];
  const float* sin = state_in ? state_in + seg * state_in_seg + (b * heads + h) * (int64_t)dim * vdim : nullptr;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (warp * MT + mt) * 16 + g8 + (e >> 1) * 8, c = c0 + nt * 8 + t4 * 2 + (e & 1);
        st[mt][nt][e] = (OUTPUT && !fresh && sin && r < dim && c < vdim) ? sin[(int64_t)r * vdim + c] : 0.f;
      }

  load_chunk(tok0, 0);
  int stage = 0;
  for (int t0 = tok0; t0 < tok1; t0 += kChunk, stage ^= 1) {
    const int n = min(kChunk, tok1 - t0);
    __syncthreads();  // everyone is done with the other stage and with the state parts of the chunk before
    if (t0 + kChunk < tok1) {
      load_chunk(t0 + kChunk, stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    if (OUTPUT) {
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
          for (int e = 0; e < 4; e += 2) {
            const int r = (warp * MT + mt) * 16 + g8 + (e >> 1) * 8;
            uint32_t hi, lo;
            split_pair(st[mt][nt][e], st[mt][nt][e + 1], hi, lo);
            const uint32_t at = swz<VROW>(r, nt) + t4 * 4;
            asm volatile("st.shared.b32 [%0], %1;" ::"r"(s_hi + at), "r"(hi) : "memory");
            asm volatile("st.shared.b32 [%0], %1;" ::"r"(s_lo + at), "r"(lo) : "memory");
          }
    }
    __syncthreads();  // tiles and state parts are in place
    const uint32_t sq = base + stage * M::STAGE_BYTES, sk = sq + M::QK_BYTES, sv = sk + M::QK_BYTES;

    if (OUTPUT) {
      // this warp's 16 tokens: rows warp * 16 + {g8, g8 + 8} of the chunk
      float o[8][4], a[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = a[i][0] = a[i][1] = a[i][2] = a[i][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DIM / 16; ++ks) {
        uint32_t qf[4];
        ldsm4(qf, sq + swz<QROW>(warp * 16 + (lane & 15), ks * 2 + (lane >> 4)));
        // scores against the chunk's keys up to this warp's last token
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          if (np <= warp) {
            uint32_t kf[4];
            ldsm4(kf, sk + swz<QROW>(np * 16 + (lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1)));
            mma_bf16(a[2 * np], qf, kf[0], kf[1]);
            mma_bf16(a[2 * np + 1], qf, kf[2], kf[3]);
          }
        }
        // q S
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          const uint32_t at = swz<VROW>(ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, np * 2 + (lane >> 4));
          uint32_t sf[4];
          ldsm4_trans(sf, s_hi + at);
          mma_bf16(o[2 * np], qf, sf[0], sf[1]);
          mma_bf16(o[2 * np + 1], qf, sf[2], sf[3]);
          ldsm4_trans(sf, s_lo + at);
          mma_bf16(o[2 * np], qf, sf[0], sf[1]);
          mma_bf16(o[2 * np + 1], qf, sf[2], sf[3]);
        }
      }
      const int i0 = warp * 16 + g8;
      // gates of this thread's outputs, on their way while the scores are applied (pairs of columns; vdim is a multiple of 8)
      uint32_t gate[2][8];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const __nv_bfloat16* src = qkvg + (b * n_tok + t0 + i0 + r * 8) * ld + off_g + (int64_t)h * vdim + c0 + t4 * 2;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
          gate[r][nt] = i0 + r * 8 < n && c0 + nt * 8 < vdim ? __ldg(reinterpret_cast<const unsigned int*>(src + nt * 8)) : 0u;
      }
      const float p0 = pw[i0 + 1], p1 = pw[i0 + 9];
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        o[nt][0] *= p0, o[nt][1] *= p0, o[nt][2] *= p1, o[nt][3] *= p1;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int age = i0 + (e >> 1) * 8 - (nt * 8 + t4 * 2 + (e & 1));
          a[nt][e] = age >= 0 ? a[nt][e] * pw[age] : 0.f;
        }
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        if (kk <= warp) {
          uint32_t ah[4], al[4];
          split_pair(a[2 * kk][0], a[2 * kk][1], ah[0], al[0]);
          split_pair(a[2 * kk][2], a[2 * kk][3], ah[1], al[1]);
          split_pair(a[2 * kk + 1][0], a[2 * kk + 1][1], ah[2], al[2]);
          split_pair(a[2 * kk + 1][2], a[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
          for (int np = 0; np < 4; ++np) {
            uint32_t vf[4];
            ldsm4_trans(vf, sv + swz<VROW>(kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, np * 2 + (lane >> 4)));
            mma_bf16(o[2 * np], ah, vf[0], vf[1]);
            mma_bf16(o[2 * np + 1], ah, vf[2], vf[3]);
            mma_bf16(o[2 * np], al, vf[0], vf[1]);
            mma_bf16(o[2 * np + 1], al, vf[2], vf[3]);
          }
        }
      }
      // o * weight * gate, and the rows' sums of squares over this block's columns
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = i0 + r * 8;
        const int64_t row = b * n_tok + t0 + t;
        float sq2 = 0.f;
        if (t < n) {
#pragma unroll
          for (int nt = 0; nt < 8; ++nt) {
            const int c = nt * 8 + t4 * 2;
            if (c0 + c < vdim) {
              const float2 gt = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gate[r][nt]));
              const float o0 = o[nt][2 * r], o1 = o[nt][2 * r + 1];
              sq2 = fmaf(o0, o0, fmaf(o1, o1, sq2));
              *reinterpret_cast<__nv_bfloat162*>(y + row * ld_y + (int64_t)h * vdim + c0 + c) = __floats2bfloat162_rn(o0 * ws[c] * gt.x, o1 * ws[c + 1] * gt.y);
            }
          }
        }
        sq2 += __shfl_xor_sync(0xffffffffu, sq2, 1);
        sq2 += __shfl_xor_sync(0xffffffffu, sq2, 2);
        if (t4 == 0 && t < n) sumsq[(int64_t)(h * vblocks + vb) * ld_sumsq + row] = sq2;
      }
    }

    // S <- decay^n S + sum_j (decay^(n-1-j) k_j) v_j^T
    const float pn = pw[n];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[mt][nt][e] *= pn;
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      // exponents of the two token pairs this thread holds (rows beyond n are zero: any finite factor will do)
      float f[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) f[i] = pw[max(0, n - 1 - (kk * 16 + t4 * 2 + (i & 1) + (i >> 1) * 8))];
      uint32_t kh[MT][4], kl[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        // K^T: rows = state rows, columns = tokens; matrices (rows 0-7, tokens 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15)
        uint32_t kf[4];
        const int piece = ((warp * MT + mt) * 16) / 8 + ((lane >> 3) & 1);
        ldsm4_trans(kf, sk + swz<QROW>(kk * 16 + (lane & 7) + ((lane >> 4) << 3), piece));
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&kf[i]));
          split_pair(x.x * f[(i >> 1) * 2], x.y * f[(i >> 1) * 2 + 1], kh[mt][i], kl[mt][i]);
        }
      }
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t vf[4];
        ldsm4_trans(vf, sv + swz<VROW>(kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, np * 2 + (lane >> 4)));
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16(st[mt][2 * np], kh[mt], vf[0], vf[1]);
          mma_bf16(st[mt][2 * np + 1], kh[mt], vf[2], vf[3]);
          mma_bf16(st[mt][2 * np], kl[mt], vf[0], vf[1]);
          mma_bf16(st[mt][2 * np + 1], kl[mt], vf[2], vf[3]);
        }
      }
    }
  }
  // the state after the segment: everyone's (first pass), or the last segment's (the sequence's new state)
  if (!OUTPUT || seg + 1 == gridDim.y) {
    float* out = state_out + seg * state_out_seg + (b * heads + h) * (int64_t)dim * vdim;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int r = (warp * MT + mt) * 16 + g8 + (e >> 1) * 8, c = c0 + nt * 8 + t4 * 2;
          if (r < dim && c < vdim) *reinterpret_cast<float2*>(out + (int64_t)r * vdim + c) = make_float2(st[mt][nt][e], st[mt][nt][e + 1]);
        }
  }
}

// added[s] (s < n_seg - 1) holds what segment s adds to the state; afterwards starts[s] is the state in front of segment s.
__global__ void __launch_bounds__(256)
segment_scan_kernel(const float* __restrict__ state, int fresh, float* __restrict__ starts, const float* __restrict__ added, int64_t stride,
                    const double* __restrict__ decay, int seg_len, int n_seg, int heads, int64_t per_head) {
  const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (i >= stride) return;
  const float f = (float)pow(decay[(i / per_head) % heads], (double)seg_len);
  float s = fresh ? 0.f : state[i];
  for (int k = 0; k < n_seg; ++k) {
    starts[(int64_t)k * stride + i] = s;
    if (k + 1 < n_seg) s = fmaf(f, s, added[(int64_t)k * stride + i]);
  }
}

bool takes_chunks(int64_t n_tok, int64_t dim, int64_t vdim, int dtype) {
  return dtype == B200_BF16 && n_tok >= kChunk / 2 && dim <= 128 && dim % 8 == 0 && vdim % 8 == 0;
}
// Segments per sequence: the fewest rounds of blocks (two per SM), counted in chunks; the first pass over all but the last
// segment costs about 0.4 of a full one, and extra launches a few chunks.
int64_t segment_count(int64_t B, int64_t n_tok, int64_t heads, int64_t vdim) {
  const int64_t blocks = B * heads * ((vdim + kVCols - 1) / kVCols), slots = (int64_t)sm_count() * 2, chunks = (n_tok + kChunk - 1) / kChunk;
  auto rounds = [&](int64_t n) { return (double)((blocks * n + slots - 1) / slots); };
  int64_t best = 1;
  double cost = rounds(1) * chunks;
  for (int64_t n = 2; n <= 64 && n * 4 <= chunks; ++n) {
    const double per = (double)((chunks + n - 1) / n), c = rounds(n) * per + 0.4 * rounds(n - 1) * per + 3.0;
    if (c < cost) cost = c, best = n;
  }
  return best;
}

template <int DIM>
int launch_chunked(const Args& a, void* workspace, cudaStream_t stream) {
  constexpr int smem = ChunkSmem<DIM>::BYTES;
  static std::atomic<bool> attr_set[kMaxDevices];
  const int slot = device_slot();
  if (slot < 0) return B200_ERR_CUDA;
  if (!attr_set[slot].load(std::memory_order_acquire)) {
    if (cudaFuncSetAttribute(chunked_kernel<DIM, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess ||
        cudaFuncSetAttribute(chunked_kernel<DIM, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return B200_ERR_CUDA;
    attr_set[slot].store(true, std::memory_order_release);
  }
  const int64_t blocks = a.B * a.heads * ((a.vdim + kVCols - 1) / kVCols);
  if (blocks > 0x7fffffffLL || a.n_tok > 0x7fffffffLL - kChunk) return B200_ERR_BAD_ARGUMENT;
  int64_t n_seg = segment_count(a.B, a.n_tok, a.heads, a.vdim);  // (the workspace is sized for this many)
  const int64_t chunks = (a.n_tok + kChunk - 1) / kChunk, per = (chunks + n_seg - 1) / n_seg;
  const int seg_len = (int)(per * kChunk);
  n_seg = (chunks + per - 1) / per;
  if (n_seg > 65535) return B200_ERR_BAD_ARGUMENT;
  const int64_t stride = a.B * a.heads * a.dim * a.vdim;
  const auto* x = static_cast<const __nv_bfloat16*>(a.qkvg);
  const float* start = a.state;
  int64_t start_seg = 0;
  int fresh = a.fresh;
  if (n_seg > 1) {
    float* added = static_cast<float*>(workspace);
    float* starts = added + (n_seg - 1) * stride;
    chunked_kernel<DIM, false><<<dim3((unsigned)blocks, (unsigned)(n_seg - 1)), kChunkThreads, smem, stream>>>(
        x, a.ld, a.off_k, a.off_v, a.off_g, a.decay, a.weight, nullptr, 0, added, stride, 1, nullptr, 0, nullptr, 0, (int)a.n_tok, seg_len, (int)a.heads,
        (int)a.dim, (int)a.vdim);
    segment_scan_kernel<<<(unsigned)((stride + 255) / 256), 256, 0, stream>>>(a.state, a.fresh, starts, added, stride, a.decay, seg_len, (int)n_seg,
                                                                              (int)a.heads, a.dim * a.vdim);
    note_launches(2);
    start = starts, start_seg = stride, fresh = 0;
  }
  chunked_kernel<DIM, true><<<dim3((unsigned)blocks, (unsigned)n_seg), kChunkThreads, smem, stream>>>(
      x, a.ld, a.off_k, a.off_v, a.off_g, a.decay, a.weight, start, start_seg, a.state, 0, fresh, static_cast<__nv_bfloat16*>(a.y), a.ld_y, a.sumsq, a.ld_sumsq,
      (int)a.n_tok, seg_len, (int)a.heads, (int)a.dim, (int)a.vdim);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

}  // namespace

int64_t decayed_attention_slices(int64_t n_tok, int64_t heads, int64_t dim, int64_t vdim, int dtype) {
  const int64_t cols = takes_chunks(n_tok, dim, vdim, dtype) ? kVCols : kCols;
  return heads * ((vdim + cols - 1) / cols);
}

size_t decayed_attention_workspace_bytes(int64_t B, int64_t n_tok, int64_t heads, int64_t dim, int64_t vdim, int dtype) {
  if (!takes_chunks(n_tok, dim, vdim, dtype)) return 0;
  const int64_t n_seg = segment_count(B, n_tok, heads, vdim);
  return n_seg < 2 ? 0 : (size_t)(2 * n_seg * B * heads * dim * vdim) * 4;
}

int launch_decayed_attention(const void* qkvg, int64_t ld, int64_t off_k, int64_t off_v, int64_t off_g, const double* decay, const float* weight,
                             float* state, int fresh, void* y, int64_t ld_y, float* sumsq, int64_t ld_sumsq, int64_t B, int64_t n_tok, int64_t heads,
                             int64_t dim, int64_t vdim, int dtype, void* workspace, int* status_word, cudaStream_t stream) {
  (void)status_word;
  const Args a{qkvg, ld, off_k, off_v, off_g, decay, weight, state, fresh, y, ld_y, sumsq, ld_sumsq, B, n_tok, heads, dim, vdim};
  // (16-byte pieces of q, k, v rows; pairs of the rest)
  const bool aligned = ((reinterpret_cast<uintptr_t>(qkvg) | reinterpret_cast<uintptr_t>(weight) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(state)) & 15) == 0 &&
                       ld % 8 == 0 && off_k % 8 == 0 && off_v % 8 == 0 && off_g % 8 == 0 && ld_y % 2 == 0;
  if (takes_chunks(n_tok, dim, vdim, dtype)) {
    if (!aligned) return B200_ERR_ALIGNMENT;
    return dim <= 64 ? launch_chunked<64>(a, workspace, stream) : launch_chunked<128>(a, workspace, stream);
  }
  return dtype == B200_BF16 ? launch_recurrent<__nv_bfloat16>(a, stream) : launch_recurrent<float>(a, stream);
}

}  // namespace b200
