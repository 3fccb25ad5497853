// Gated delta rule over many tokens, bf16, 64 tokens at a time on the tensor cores (mma.sync: the dependent chain of a
// chunk is short products of 64 rows).  With S the state before a chunk, G_i the product of the decays up to token i of the
// chunk, c_k and c_q the convolved keys and queries and r_k, r_q what makes them unit vectors (and scales q):
//     A_ij = beta_i (G_i / G_j) r_ki r_kj (c_ki . c_kj), j < i        T = (I + A)^-1 diag(beta)
//     P_ij = (G_i / G_j) r_qi r_kj (c_qi . c_kj), j <= i
//     U = T (V - diag(G r_k) C_k S)                                   what the tokens write
//     O = diag(G r_q) C_q S + P U
//     S <- G_64 S + C_k^T diag((G_64 / G_j) r_kj) U
// Every ratio of decays has j <= i: nothing overflows, whatever the decays.  c_q, c_k and v are bf16 and enter the MMAs as
// they are; what is fp32 by definition (S, T, P, U and V - ...) enters as two bf16 parts (16 bits) and is accumulated in fp32.
//
//   delta_conv_kernel     convolution and silu, 32 tokens x 8 channels per thread
//   delta_chunk_prepare   per (chunk, head), in parallel: gates, unit norms, A, its triangular inverse, P; T and P leave in
//                         the register layout of the MMAs that read them
//   delta_chunk_scan      per (sequence, head, column block): the chunks one after the other, S in registers
//   delta_finish_kernel   norm per head and gate
#include <atomic>

#include "mma_sync.cuh"
#include "sm100_primitives.cuh"

namespace b200 {
namespace {

using namespace warp_mma;

constexpr int kC = 64;  // tokens per chunk

// ------------------------------------------------------------------ convolution and silu
constexpr int kConvTokens = 32, kConvBatch = 8;  // tokens per thread, loads in flight
// a / (1 + exp(-a)) with one ex2 and one reciprocal
__device__ __forceinline__ float silu_quick(float a) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(a * -1.4426950408889634f));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
  return a * r;
}
// One thread: 8 channels of kConvTokens tokens of one sequence; the last TAPS - 1 inputs stay in registers.
template <int TAPS>
__global__ void __launch_bounds__(128)
delta_conv_kernel(b200_delta_args p, int vecs) {
  const int v = blockIdx.x * 128 + threadIdx.x;
  if (v >= vecs) return;
  const int64_t c = (int64_t)v * 8, b = blockIdx.z, t0 = (int64_t)blockIdx.y * kConvTokens;
  const auto* rows = static_cast<const __nv_bfloat16*>(p.rows) + b * p.n * p.ld + c;
  auto* out = static_cast<__nv_bfloat16*>(p.mixed) + b * p.n * p.ld_mixed + c;
  const auto* ring = static_cast<const __nv_bfloat16*>(p.conv_state) + b * p.taps * p.conv_cols + c;
  float2 w[TAPS][4], x[TAPS][4];  // pairs of channels: packed multiply-adds
  {
    float f[8 * TAPS];  // (8 * TAPS consecutive floats from a multiple of 32 bytes on)
#pragma unroll
    for (int i = 0; i < 8 * TAPS; i += 4) {
      const float4 v4 = __ldg(reinterpret_cast<const float4*>(p.conv_w + c * TAPS + i));
      f[i] = v4.x, f[i + 1] = v4.y, f[i + 2] = v4.z, f[i + 3] = v4.w;
    }
#pragma unroll
    for (int k = 0; k < TAPS; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) w[k][e] = make_float2(f[2 * e * TAPS + k], f[(2 * e + 1) * TAPS + k]);
  }
  auto unpack = [](const uint4& u, float2 (&f)[4]) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int e = 0; e < 4; ++e) f[e] = __bfloat1622float2(h[e]);
  };
  auto load = [&](const __nv_bfloat16* src, bool ok) { return ok ? __ldg(reinterpret_cast<const uint4*>(src)) : make_uint4(0, 0, 0, 0); };
#pragma unroll
  for (int k = 0; k < TAPS - 1; ++k) {
    const int64_t t = t0 - (TAPS - 1) + k, pos = p.start + t;
    unpack(t >= 0 ? load(rows + t * p.ld, true) : load(ring + (pos + TAPS) % TAPS * p.conv_cols, pos >= 0), x[k]);
  }
  for (int i0 = 0; i0 < kConvTokens; i0 += kConvBatch) {
    uint4 raw[kConvBatch];
#pragma unroll
    for (int i = 0; i < kConvBatch; ++i) raw[i] = load(rows + (t0 + i0 + i) * p.ld, t0 + i0 + i < p.n);
#pragma unroll
    for (int i = 0; i < kConvBatch; ++i) {
      const int64_t t = t0 + i0 + i;
      unpack(raw[i], x[TAPS - 1]);
      uint4 res;
      uint32_t* o = reinterpret_cast<uint32_t*>(&res);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float2 a = __fmul2_rn(w[0][e], x[0][e]);
#pragma unroll
        for (int k = 1; k < TAPS; ++k) a = __ffma2_rn(w[k][e], x[k][e], a);
        const __nv_bfloat162 h = __floats2bfloat162_rn(silu_quick(a.x), silu_quick(a.y));
        o[e] = *reinterpret_cast<const uint32_t*>(&h);
      }
      if (t < p.n) *reinterpret_cast<uint4*>(out + t * p.ld_mixed) = res;
#pragma unroll
      for (int k = 0; k + 1 < TAPS; ++k)
#pragma unroll
        for (int e = 0; e < 4; ++e) x[k][e] = x[k + 1][e];
    }
  }
}
template <int TAPS>
int launch_conv(const b200_delta_args& p, cudaStream_t stream) {
  const int vecs = (int)(p.conv_cols / 8);
  delta_conv_kernel<TAPS><<<dim3((unsigned)((vecs + 127) / 128), (unsigned)((p.n + kConvTokens - 1) / kConvTokens), (unsigned)p.B), 128, 0, stream>>>(p, vecs);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

// ------------------------------------------------------------------ per chunk and head, in parallel
// What a (chunk, head) leaves for the scan: T and P as A fragments of m16n8k16 (the ten 16 x 16 blocks on and below the
// diagonal, high parts then low parts, 512 bytes each), four fp32 factors per token, and the chunk's decay.
constexpr int kBlocks = 10, kFragBytes = kBlocks * 2 * 512;
constexpr int kFactorBytes = 4 * kC * 4;  // [G r_k | G r_q | (G_64 / G) r_k | unused]
constexpr int kRecordBytes = 2 * kFragBytes + kFactorBytes + 64;
enum { F_GK = 0, F_GQ = 1, F_WRITE = 2 };
__device__ __forceinline__ int block_index(int mt, int kt) { return mt * (mt + 1) / 2 + kt; }

template <int DIM>
struct PrepareSmem {
  static constexpr int PITCH = DIM * 2 + 16;  // bytes per row of a token tile: ldmatrix rows fall into different banks
  static constexpr int TILE = kC * PITCH;
  static constexpr int A_PITCH = kC + 4;      // floats
  static constexpr int SQUARE = kC * A_PITCH * 4;  // A and its inverse take the tiles' place
  static constexpr int BYTES = 2 * (TILE > SQUARE ? TILE : SQUARE);
};

__device__ __forceinline__ float ex2_ratio(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Rows of 16-byte pieces of one head's columns, zero beyond the last token and column.
template <int DIM>
__device__ __forceinline__ void load_tile(uint32_t dst, const __nv_bfloat16* src, int64_t ld, int n, int cols, int thread, int threads) {
  constexpr int PITCH = DIM * 2 + 16;
  for (int i = thread; i < kC * (DIM / 8); i += threads) {
    const int r = i / (DIM / 8), c = i % (DIM / 8);
    const bool ok = r < n && c * 8 < cols;
    cp_async16(dst + r * PITCH + c * 16, ok ? src + (int64_t)r * ld + c * 8 : src, ok);
  }
}

template <int DIM>
__global__ void __launch_bounds__(128)
delta_chunk_prepare(b200_delta_args p, int n_chunks) {
  using M = PrepareSmem<DIM>;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float cum_hi[kC], cum_lo[kC], beta_s[kC], rk_s[kC], rq_s[kC];
  __shared__ double warp_total;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
  const int64_t h = blockIdx.x % p.heads, chunk = (blockIdx.x / p.heads) % n_chunks, b = blockIdx.x / (p.heads * n_chunks);
  const int64_t kv = h / (p.heads / p.kv_heads), t0 = chunk * kC, row0 = b * p.n + t0;
  const int n = (int)(p.n - t0 < kC ? p.n - t0 : kC);
  uint8_t* record = static_cast<uint8_t*>(p.workspace) + (int64_t)blockIdx.x * kRecordBytes;
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem), sq = base, sk = base + M::TILE;
  float* A = reinterpret_cast<float*>(smem);  // [64][68]
  float* X = A + kC * M::A_PITCH;             // its inverse
  const auto* mixed = static_cast<const __nv_bfloat16*>(p.mixed) + row0 * p.ld_mixed + kv * p.dim;
  load_tile<DIM>(sq, mixed, p.ld_mixed, n, (int)p.dim, threadIdx.x, 128);
  load_tile<DIM>(sk, mixed + p.off_k, p.ld_mixed, n, (int)p.dim, threadIdx.x, 128);
  cp_async_commit();
  // log2 decays, their running sum in two fp32 parts (differences stay exact however long and strong the decays), step sizes
  if (threadIdx.x < kC) {
    const int i = threadIdx.x;
    double s = 0.0;
    float beta = 0.f;
    if (i < n) {
      const auto* src = static_cast<const __nv_bfloat16*>(p.rows) + (row0 + i) * p.ld;
      const float x = __bfloat162float(src[p.off_a + h]) + p.dt_bias[h];
      s = (double)(-expf(p.a_log[h]) * (fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))))) * 1.4426950408889634;
      beta = 1.0f / (1.0f + expf(-__bfloat162float(src[p.off_b + h])));
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double before = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += before;
    }
    if (i == 31) warp_total = s;
    asm volatile("bar.sync 1, 64;" ::: "memory");
    if (i >= 32) s += warp_total;
    const float hi = (float)s;
    cum_hi[i] = hi, cum_lo[i] = (float)(s - (double)hi);
    beta_s[i] = beta;
  }
  cp_async_wait<0>();
  __syncthreads();
  // unit norms of the stored rows: two threads per row
  {
    const int r = threadIdx.x >> 1, side = threadIdx.x & 1;
    float a = 0.f, c = 0.f;
    for (int i = side * 8; i < DIM; i += 16) {
      float f[8];
      load8(reinterpret_cast<const __nv_bfloat16*>(smem + r * M::PITCH + i * 2), f);
#pragma unroll
      for (int e = 0; e < 8; ++e) a = fmaf(f[e], f[e], a);
      load8(reinterpret_cast<const __nv_bfloat16*>(smem + M::TILE + r * M::PITCH + i * 2), f);
#pragma unroll
      for (int e = 0; e < 8; ++e) c = fmaf(f[e], f[e], c);
    }
    a += __shfl_xor_sync(0xffffffffu, a, 1);
    c += __shfl_xor_sync(0xffffffffu, c, 1);
    if (side == 0) rq_s[r] = p.q_scale / sqrtf(a + p.unit_eps), rk_s[r] = 1.0f / sqrtf(c + p.unit_eps);
  }
  __syncthreads();
  // this warp's 16 rows of C_k C_k^T and C_q C_k^T, up to its last token
  float kk[8][4], qk[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) kk[i][e] = qk[i][e] = 0.f;
#pragma unroll
  for (int ks = 0; ks < DIM / 16; ++ks) {
    uint32_t qf[4], kf[4];
    const uint32_t at = (uint32_t)((warp * 16 + (lane & 15)) * M::PITCH + (ks * 2 + (lane >> 4)) * 16);
    ldsm4(qf, sq + at);
    ldsm4(kf, sk + at);
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      if (np <= warp) {
        uint32_t bf[4];
        ldsm4(bf, sk + (uint32_t)((np * 16 + (lane & 7) + ((lane >> 4) << 3)) * M::PITCH + (ks * 2 + ((lane >> 3) & 1)) * 16));
        mma_bf16(kk[2 * np], kf, bf[0], bf[1]);
        mma_bf16(kk[2 * np + 1], kf, bf[2], bf[3]);
        mma_bf16(qk[2 * np], qf, bf[0], bf[1]);
        mma_bf16(qk[2 * np + 1], qf, bf[2], bf[3]);
      }
    }
  }
  __syncthreads();  // the tiles are done with
  const int i0 = warp * 16 + g8;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = i0 + r * 8;
    const float hi = cum_hi[i], lo = cum_lo[i], bk = beta_s[i] * rk_s[i], rq = rq_s[i];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
      if (nt / 2 > warp) continue;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int j = nt * 8 + t4 * 2 + e;
        const float f = j <= i ? ex2_ratio((hi - cum_hi[j]) + (lo - cum_lo[j])) * rk_s[j] : 0.f;
        qk[nt][2 * r + e] *= f * rq;
        A[i * M::A_PITCH + j] = j < i ? kk[nt][2 * r + e] * f * bk : 0.f;
      }
    }
  }
  // P leaves straight from the accumulators, which are laid out like an A operand
  {
    uint4* out = reinterpret_cast<uint4*>(record + kFragBytes);
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      if (kt <= warp) {
        uint4 hi, lo;
        split_pair(qk[2 * kt][0], qk[2 * kt][1], hi.x, lo.x);
        split_pair(qk[2 * kt][2], qk[2 * kt][3], hi.y, lo.y);
        split_pair(qk[2 * kt + 1][0], qk[2 * kt + 1][1], hi.z, lo.z);
        split_pair(qk[2 * kt + 1][2], qk[2 * kt + 1][3], hi.w, lo.w);
        const int at = block_index(warp, kt) * 64 + lane;
        out[at] = hi, out[at + 32] = lo;
      }
    }
  }
  __syncthreads();
  // (I + A)^-1: the two diagonal 32 x 32 blocks by forward substitution, a lane per column, ...
  if (warp < 2) {
    const float* L = A + warp * 32 * (M::A_PITCH + 1);
    float x[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      float s0 = i == lane ? 1.f : 0.f, s1 = 0.f;
#pragma unroll
      for (int j = 0; j < i; j += 4) {
        const float4 l = *reinterpret_cast<const float4*>(L + i * M::A_PITCH + j);
        s0 = fmaf(-l.x, x[j], s0);
        if (j + 1 < i) s1 = fmaf(-l.y, x[j + 1], s1);
        if (j + 2 < i) s0 = fmaf(-l.z, x[j + 2], s0);
        if (j + 3 < i) s1 = fmaf(-l.w, x[j + 3], s1);
      }
      x[i] = s0 + s1;
      X[(warp * 32 + i) * M::A_PITCH + warp * 32 + lane] = x[i];
    }
  }
  __syncthreads();
  // ... and the block below: -T22 (A21 T11).  A thread takes a 2 x 4 piece; the first product goes over A's upper right block.
  {
    const int r = (threadIdx.x >> 3) * 2, c = (threadIdx.x & 7) * 4;
    auto product = [&](const float* lhs, const float* rhs, float (&acc)[2][4]) {
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[0][e] = acc[1][e] = 0.f;
#pragma unroll 2
      for (int k = 0; k < 32; k += 4) {
        const float4 a0 = *reinterpret_cast<const float4*>(lhs + r * M::A_PITCH + k), a1 = *reinterpret_cast<const float4*>(lhs + (r + 1) * M::A_PITCH + k);
        const float l0[4] = {a0.x, a0.y, a0.z, a0.w}, l1[4] = {a1.x, a1.y, a1.z, a1.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 v = *reinterpret_cast<const float4*>(rhs + (k + i) * M::A_PITCH + c);
          acc[0][0] = fmaf(l0[i], v.x, acc[0][0]), acc[0][1] = fmaf(l0[i], v.y, acc[0][1]), acc[0][2] = fmaf(l0[i], v.z, acc[0][2]), acc[0][3] = fmaf(l0[i], v.w, acc[0][3]);
          acc[1][0] = fmaf(l1[i], v.x, acc[1][0]), acc[1][1] = fmaf(l1[i], v.y, acc[1][1]), acc[1][2] = fmaf(l1[i], v.z, acc[1][2]), acc[1][3] = fmaf(l1[i], v.w, acc[1][3]);
        }
      }
    };
    float acc[2][4];
    product(A + 32 * M::A_PITCH, X, acc);
    float* mid = A + 32;  // rows 0-31, columns 32-63
#pragma unroll
    for (int e = 0; e < 2; ++e) *reinterpret_cast<float4*>(mid + (r + e) * M::A_PITCH + c) = make_float4(acc[e][0], acc[e][1], acc[e][2], acc[e][3]);
    __syncthreads();
    product(X + 32 * (M::A_PITCH + 1), mid, acc);
#pragma unroll
    for (int e = 0; e < 2; ++e)
      *reinterpret_cast<float4*>(X + (32 + r + e) * M::A_PITCH + c) = make_float4(-acc[e][0], -acc[e][1], -acc[e][2], -acc[e][3]);
  }
  __syncthreads();
  {
    uint4* out = reinterpret_cast<uint4*>(record);
    const int mt = warp;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      if (kt <= mt) {
        const int c = kt * 16 + t4 * 2;
        // (inside a diagonal block of 32 the substitution wrote its zeros above the diagonal)
        auto pair = [&](int row, int col) {
          const float2 v = *reinterpret_cast<const float2*>(X + row * M::A_PITCH + col);
          return make_float2(v.x * beta_s[col], v.y * beta_s[col + 1]);
        };
        const float2 a = pair(mt * 16 + g8, c), d = pair(mt * 16 + g8 + 8, c), e = pair(mt * 16 + g8, c + 8), f = pair(mt * 16 + g8 + 8, c + 8);
        uint4 hi, lo;
        split_pair(a.x, a.y, hi.x, lo.x);
        split_pair(d.x, d.y, hi.y, lo.y);
        split_pair(e.x, e.y, hi.z, lo.z);
        split_pair(f.x, f.y, hi.w, lo.w);
        const int at = block_index(mt, kt) * 64 + lane;
        out[at] = hi, out[at + 32] = lo;
      }
    }
  }
  float* factor = reinterpret_cast<float*>(record + 2 * kFragBytes);
  if (threadIdx.x < kC) {
    const int i = threadIdx.x;
    const float G = ex2_ratio(cum_hi[i] + cum_lo[i]);
    factor[F_GK * kC + i] = G * rk_s[i];
    factor[F_GQ * kC + i] = G * rq_s[i];
    factor[F_WRITE * kC + i] = i < n ? ex2_ratio((cum_hi[kC - 1] - cum_hi[i]) + (cum_lo[kC - 1] - cum_lo[i])) * rk_s[i] : 0.f;
    if (i == kC - 1) factor[4 * kC] = G;
  }
}

// ------------------------------------------------------------------ chunk after chunk
// A block owns VC columns of one head's state.  Half of its warps run the chain from state to state (C_k S -> R -> U -> S), the
// other half the outputs beside it; each half is 4 row groups x (VC / CW) column groups of CW columns.
template <int DIM, int VC, int CW>
struct ScanSmem {
  static constexpr int ROLE_WARPS = 4 * (VC / CW), THREADS = 64 * ROLE_WARPS;
  // a stage: keys, queries (DIM / 64 TMA atoms of 64 rows x 128 bytes each, 128-byte swizzle), 64 columns of values, the record
  static constexpr int ATOM = kC * 128, TILE = DIM / 64 * ATOM;
  static constexpr int V_AT = 2 * TILE, RECORD_AT = V_AT + ATOM, FACTOR_AT = RECORD_AT + 2 * kFragBytes;
  static constexpr int STAGE = (RECORD_AT + kRecordBytes + 1023) / 1024 * 1024, STAGES = VC == 16 ? 3 : 2;
  static constexpr int TX_BYTES = 2 * TILE + ATOM + kRecordBytes;
  static constexpr int VP = VC * 2 + 16;  // bytes per row of the tiles below: ldmatrix rows fall into different banks
  static constexpr int V_TILE = kC * VP, S_PART = DIM * VP;
  static constexpr int BYTES = STAGES * STAGE + 2 * S_PART + 6 * V_TILE + 1024;  // S, R, U, U' in two parts each; alignment
};

// size a multiple of 16 bytes, both addresses 16-byte aligned
__device__ __forceinline__ void bulk_copy(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

template <int DIM, int VC, int CW>
__global__ void __launch_bounds__(ScanSmem<DIM, VC, CW>::THREADS, 1)
delta_chunk_scan(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, b200_delta_args p,
                 int n_chunks, int vblocks) {
  using M = ScanSmem<DIM, VC, CW>;
  constexpr int MT = DIM / 64, NT = CW / 8;  // 16-row state tiles per warp, 8-column tiles per warp
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t full[M::STAGES];  // a stage's copies have landed
  __shared__ volatile int aborted;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
  const bool chain = warp < M::ROLE_WARPS;
  // row group, column group; every other four warps in reverse, so that a scheduler's warps share the triangles' work evenly
  const int cg = (warp % M::ROLE_WARPS) >> 2, rg = ((warp >> 2) & 1) ? 3 - (warp & 3) : warp & 3;
  const int vb = blockIdx.x % vblocks;
  const int64_t h = (blockIdx.x / vblocks) % p.heads, b = blockIdx.x / ((int64_t)vblocks * p.heads);
  const int64_t kv = h / (p.heads / p.kv_heads);
  const int c0 = vb * VC, dim = (int)p.dim, vdim = (int)p.vdim;
  const uint32_t raw = (uint32_t)__cvta_generic_to_shared(smem_raw), base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (base - raw);
  const uint32_t s_hi = base + M::STAGES * M::STAGE, s_lo = s_hi + M::S_PART;
  const uint32_t r_hi = s_lo + M::S_PART, r_lo = r_hi + M::V_TILE, u_hi = r_lo + M::V_TILE, u_lo = u_hi + M::V_TILE, w_hi = u_lo + M::V_TILE, w_lo = w_hi + M::V_TILE;
  const uint8_t* records = static_cast<const uint8_t*>(p.workspace) + (b * n_chunks * p.heads + h) * (int64_t)kRecordBytes;
  const int64_t record_step = p.heads * (int64_t)kRecordBytes;
  const int i0 = rg * 16 + g8;  // this thread's tokens of a chunk: i0 and i0 + 8

  const uint32_t bar_full = (uint32_t)__cvta_generic_to_shared(full);
  if (threadIdx.x == 0) {
    for (int i = 0; i < M::STAGES; ++i) sm100::mbar_init(bar_full + 8 * i, 1);
    aborted = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    sm100::fence_proxy_async_smem();
  }
  __syncthreads();
  // one thread (rows behind the last token and columns beyond a head arrive as zeros)
  auto load_chunk = [&](int chunk, int stage) {
    const uint32_t dst = base + stage * M::STAGE, bar = bar_full + 8 * stage;
    sm100::mbar_arrive_expect_tx(bar, M::TX_BYTES);
#pragma unroll
    for (int a = 0; a < DIM / 64; ++a) {
      sm100::tma_load_4d(dst + a * M::ATOM, &map_k, bar, 64 * a, (int)kv, chunk * kC, (int)b);
      sm100::tma_load_4d(dst + M::TILE + a * M::ATOM, &map_q, bar, 64 * a, (int)kv, chunk * kC, (int)b);
    }
    sm100::tma_load_4d(dst + M::V_AT, &map_v, bar, c0, (int)h, chunk * kC, (int)b);
    bulk_copy(dst + M::RECORD_AT, records + chunk * record_step, kRecordBytes, bar);
  };
  // address of a 16-byte piece of a row of keys or queries
  auto piece_at = [](uint32_t tile, int row, int piece) { return tile + (uint32_t)((piece >> 3) * M::ATOM) + swz<128>(row, piece & 7); };
  // accumulators (rows of 16, this warp's columns) as two bf16 parts into a row-major tile
  auto put = [&](uint32_t hi, uint32_t lo, int row, int nt, float a, float c) {
    uint32_t x, y;
    split_pair(a, c, x, y);
    const uint32_t at = (uint32_t)(row * M::VP + (cg * CW + nt * 8 + t4 * 2) * 2);
    asm volatile("st.shared.b32 [%0], %1;" ::"r"(hi + at), "r"(x) : "memory");
    asm volatile("st.shared.b32 [%0], %1;" ::"r"(lo + at), "r"(y) : "memory");
  };
  // address of a B fragment (16 rows of k from `row`, 16 columns from np * 16 of this warp's)
  auto b_at = [&](int row, int np) {
    return (uint32_t)((row + (lane & 7) + ((lane >> 3) & 1) * 8) * M::VP + (cg * CW + np * 16 + (lane >> 4) * 8) * 2);
  };
  // acc = 64 token rows (this warp's 16) times the state in two parts
  auto times_state = [&](uint32_t tile, float (&acc)[NT][4]) {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DIM / 16; ++ks) {
      uint32_t af[4];
      ldsm4(af, piece_at(tile, rg * 16 + (lane & 15), ks * 2 + (lane >> 4)));
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        uint32_t hi[4], lo[4];
        const uint32_t bt = b_at(ks * 16, np);
        ldsm4_trans(hi, s_hi + bt);
        ldsm4_trans(lo, s_lo + bt);
        mma_bf16(acc[2 * np], af, hi[0], hi[1]);
        mma_bf16(acc[2 * np + 1], af, hi[2], hi[3]);
        mma_bf16(acc[2 * np], af, lo[0], lo[1]);
        mma_bf16(acc[2 * np + 1], af, lo[2], lo[3]);
      }
    }
  };
  // acc += T (which = 0) or P (1) of the stage's record times a tile in two parts, for this warp's rows
  auto triangular = [&](int stage, int which, uint32_t hi_tile, uint32_t lo_tile, float (&acc)[NT][4]) {
    const uint4* frag = reinterpret_cast<const uint4*>(smem + stage * M::STAGE + M::RECORD_AT + which * kFragBytes) + block_index(rg, 0) * 64 + lane;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      if (kt <= rg) {
        const uint4 ah = frag[kt * 64], al = frag[kt * 64 + 32];
        const uint32_t fh[4] = {ah.x, ah.y, ah.z, ah.w}, fl[4] = {al.x, al.y, al.z, al.w};
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          uint32_t hi[4], lo[4];
          const uint32_t bt = b_at(kt * 16, np);
          ldsm4_trans(hi, hi_tile + bt);
          ldsm4_trans(lo, lo_tile + bt);
          mma_bf16(acc[2 * np], fh, hi[0], hi[1]);
          mma_bf16(acc[2 * np + 1], fh, hi[2], hi[3]);
          mma_bf16(acc[2 * np], fl, hi[0], hi[1]);
          mma_bf16(acc[2 * np + 1], fl, hi[2], hi[3]);
          mma_bf16(acc[2 * np], fh, lo[0], lo[1]);
          mma_bf16(acc[2 * np + 1], fh, lo[2], lo[3]);
        }
      }
    }
  };

  int stage = 0;
  if (chain) {
    // this warp's state: rows (rg * MT + mt) * 16 + {g8, g8 + 8}, columns cg * CW + nt * 8 + t4 * 2 + {0, 1} of the block's
    float st[MT][NT][4];
    float* state = p.state + (b * p.heads + h) * (int64_t)dim * vdim;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = (rg * MT + mt) * 16 + g8 + (e >> 1) * 8, c = c0 + cg * CW + nt * 8 + t4 * 2 + (e & 1);
          st[mt][nt][e] = !p.fresh && r < dim && c < vdim ? state[(int64_t)r * vdim + c] : 0.f;
        }
    for (int chunk = 0; chunk < n_chunks; ++chunk, stage = stage + 1 == M::STAGES ? 0 : stage + 1) {
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const int r = (rg * MT + mt) * 16 + g8;
          put(s_hi, s_lo, r, nt, st[mt][nt][0], st[mt][nt][1]);
          put(s_hi, s_lo, r + 8, nt, st[mt][nt][2], st[mt][nt][3]);
        }
      __syncthreads();  // (1) tiles and state parts are in place; everyone is done with the chunk before
      const uint32_t sk = base + stage * M::STAGE;
      const uint8_t* sv = smem + stage * M::STAGE + M::V_AT;
      const float* factor = reinterpret_cast<const float*>(smem + stage * M::STAGE + M::FACTOR_AT);
      // R = V - diag(G r_k) C_k S
      float r[NT][4];
      times_state(sk, r);
      {
        const float g0 = factor[F_GK * kC + i0], g1 = factor[F_GK * kC + i0 + 8];
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const int c = cg * CW + nt * 8 + t4 * 2;
          const float2 v0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sv + swz<128>(i0, c >> 3) + (c & 7) * 2));
          const float2 v1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sv + swz<128>(i0 + 8, c >> 3) + (c & 7) * 2));
          put(r_hi, r_lo, i0, nt, fmaf(-g0, r[nt][0], v0.x), fmaf(-g0, r[nt][1], v0.y));
          put(r_hi, r_lo, i0 + 8, nt, fmaf(-g1, r[nt][2], v1.x), fmaf(-g1, r[nt][3], v1.y));
        }
      }
      __syncthreads();  // (2) R is in place
      // U = T R, as it is for the outputs and times (G_64 / G_j) r_kj for the state
#pragma unroll
      for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) r[i][e] = 0.f;
      triangular(stage, 0, r_hi, r_lo, r);
      {
        const float f0 = factor[F_WRITE * kC + i0], f1 = factor[F_WRITE * kC + i0 + 8];
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          put(w_hi, w_lo, i0, nt, r[nt][0] * f0, r[nt][1] * f0);
          put(w_hi, w_lo, i0 + 8, nt, r[nt][2] * f1, r[nt][3] * f1);
          put(u_hi, u_lo, i0, nt, r[nt][0], r[nt][1]);
          put(u_hi, u_lo, i0 + 8, nt, r[nt][2], r[nt][3]);
        }
      }
      __syncthreads();  // (3) U and U' are in place
      // S <- G_64 S + C_k^T U'
      const float decay = factor[4 * kC];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) st[mt][nt][e] *= decay;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t kf[MT][4];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
          ldsm4_trans(kf[mt], piece_at(sk, kk * 16 + (lane & 7) + ((lane >> 4) << 3), (rg * MT + mt) * 2 + ((lane >> 3) & 1)));
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          uint32_t hi[4], lo[4];
          const uint32_t bt = b_at(kk * 16, np);
          ldsm4_trans(hi, w_hi + bt);
          ldsm4_trans(lo, w_lo + bt);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma_bf16(st[mt][2 * np], kf[mt], hi[0], hi[1]);
            mma_bf16(st[mt][2 * np + 1], kf[mt], hi[2], hi[3]);
            mma_bf16(st[mt][2 * np], kf[mt], lo[0], lo[1]);
            mma_bf16(st[mt][2 * np + 1], kf[mt], lo[2], lo[3]);
          }
        }
      }
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int r = (rg * MT + mt) * 16 + g8 + (e >> 1) * 8, c = c0 + cg * CW + nt * 8 + t4 * 2;
          if (r < dim && c < vdim) *reinterpret_cast<float2*>(state + (int64_t)r * vdim + c) = make_float2(st[mt][nt][e], st[mt][nt][e + 1]);
        }
  } else {
    const bool loads = warp == M::ROLE_WARPS && lane == 0;
    if (loads)
      for (int i = 0; i < M::STAGES - 1 && i < n_chunks; ++i) load_chunk(i, i);
    for (int chunk = 0; chunk < n_chunks; ++chunk, stage = stage + 1 == M::STAGES ? 0 : stage + 1) {
      const int64_t t0 = (int64_t)chunk * kC;
      const int n = (int)(p.n - t0 < kC ? p.n - t0 : kC);
      // (a copy that never lands would be reported through the status word; the barriers are kept up either way)
      sm100::mbar_wait(bar_full + 8 * stage, (uint32_t)(chunk / M::STAGES) & 1, &aborted, p.status_word, 81);
      __syncthreads();  // (1)
      if (loads && chunk + M::STAGES - 1 < n_chunks) load_chunk(chunk + M::STAGES - 1, stage == 0 ? M::STAGES - 1 : stage - 1);
      const float* factor = reinterpret_cast<const float*>(smem + stage * M::STAGE + M::FACTOR_AT);
      // O = diag(G r_q) C_q S + P U
      float o[NT][4];
      times_state(base + stage * M::STAGE + M::TILE, o);
      const float q0 = factor[F_GQ * kC + i0], q1 = factor[F_GQ * kC + i0 + 8];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) o[nt][0] *= q0, o[nt][1] *= q0, o[nt][2] *= q1, o[nt][3] *= q1;
      __syncthreads();  // (2)
      __syncthreads();  // (3)
      triangular(stage, 1, u_hi, u_lo, o);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = i0 + e * 8;
        if (i < n) {
          auto* y = static_cast<__nv_bfloat16*>(p.y) + (b * p.n + t0 + i) * p.ld_y + h * vdim + c0;
#pragma unroll
          for (int nt = 0; nt < NT; ++nt) {
            const int c = cg * CW + nt * 8 + t4 * 2;
            if (c0 + c < vdim) *reinterpret_cast<__nv_bfloat162*>(y + c) = __floats2bfloat162_rn(o[nt][2 * e], o[nt][2 * e + 1]);
          }
        }
      }
    }
  }
  if (aborted) {  // give copies in flight time to land before the shared memory goes away
    const long long t = clock64();
    while (clock64() - t < 2000000LL) {
    }
  }
}

// ------------------------------------------------------------------ norm per head, gate
// In place on y.  `lanes` (a power of two) lanes of 8 columns side by side take a (row, head); heads beyond 256 columns: NV = 2.
constexpr int kFinishItems = 2;  // per lane group, all loads in flight
template <int NV>
__global__ void __launch_bounds__(256)
delta_finish_kernel(b200_delta_args p, int64_t items, int lanes) {
  const int lane = threadIdx.x & 31, per_warp = 32 / lanes;
  const int64_t first = ((int64_t)blockIdx.x * 8 + (threadIdx.x >> 5)) * per_warp * kFinishItems + lane / lanes;
  const int c = (lane % lanes) * 8, vdim = (int)p.vdim, heads = (int)p.heads;
  uint4 y[kFinishItems][NV], g[kFinishItems][NV];
  int64_t at[kFinishItems];
#pragma unroll
  for (int i = 0; i < kFinishItems; ++i) {
    const int64_t item = first + i * per_warp;
    const uint32_t r32 = (uint32_t)item / (uint32_t)heads;  // (the host keeps the items below 2^31)
    const int64_t row = r32;
    const int h = (int)((uint32_t)item - r32 * (uint32_t)heads);
    at[i] = item < items ? row * p.ld_y + h * vdim + c : -1;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const bool ok = item < items && c + n * 256 < vdim;
      y[i][n] = ok ? *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.y) + at[i] + n * 256) : make_uint4(0, 0, 0, 0);
      g[i][n] = ok ? __ldg(reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.rows) + row * p.ld + p.off_g + h * vdim + c + n * 256)) : make_uint4(0, 0, 0, 0);
    }
  }
#pragma unroll
  for (int i = 0; i < kFinishItems; ++i) {
    float f[NV][8], sq = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      load8(reinterpret_cast<const __nv_bfloat16*>(&y[i][n]), f[n]);
#pragma unroll
      for (int e = 0; e < 8; ++e) sq = fmaf(f[n][e], f[n][e], sq);
    }
    for (int o = 1; o < lanes; o <<= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    const float inv = 1.0f / sqrtf(sq / (float)vdim + p.eps);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      if (at[i] >= 0 && c + n * 256 < vdim) {
        float w[8], gate[8];
        load8(p.norm_w + c + n * 256, w);
        load8(reinterpret_cast<const __nv_bfloat16*>(&g[i][n]), gate);
#pragma unroll
        for (int e = 0; e < 8; ++e) w[e] *= f[n][e] * inv * gate[e];
        store8(static_cast<__nv_bfloat16*>(p.y) + at[i] + n * 256, w);
      }
    }
  }
}
int launch_finish(const b200_delta_args& p, cudaStream_t stream) {
  int lanes = 1;
  while (lanes < 32 && lanes * 8 < p.vdim) lanes *= 2;
  const int64_t items = p.B * p.n * p.heads, per_block = 8LL * (32 / lanes) * kFinishItems;
  const unsigned grid = (unsigned)((items + per_block - 1) / per_block);
  if (p.vdim <= 256) delta_finish_kernel<1><<<grid, 256, 0, stream>>>(p, items, lanes);
  else delta_finish_kernel<2><<<grid, 256, 0, stream>>>(p, items, lanes);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

template <typename K>
bool opt_in(K* kernel, int bytes, std::atomic<bool>* done) {
  const int slot = device_slot();
  if (slot < 0) return false;
  if (done[slot].load(std::memory_order_acquire)) return true;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) != cudaSuccess) return false;
  done[slot].store(true, std::memory_order_release);
  return true;
}

template <int DIM, int VC, int CW>
int launch_scan(const b200_delta_args& p, int n_chunks, cudaStream_t stream) {
  using M = ScanSmem<DIM, VC, CW>;
  static_assert(M::BYTES <= 227 * 1024, "shared memory budget");
  static std::atomic<bool> done[kMaxDevices];
  if (!opt_in(delta_chunk_scan<DIM, VC, CW>, M::BYTES, done)) return B200_ERR_CUDA;
  const int vblocks = (int)((p.vdim + VC - 1) / VC);
  const auto* mixed = static_cast<const __nv_bfloat16*>(p.mixed);
  CUtensorMap mq, mk, mv;
  auto map = [&](CUtensorMap* m, const void* ptr, int64_t cols, int64_t heads) {
    const uint64_t dims[4] = {(uint64_t)cols, (uint64_t)heads, (uint64_t)p.n, (uint64_t)p.B};
    const uint64_t strides[3] = {(uint64_t)cols * 2, (uint64_t)p.ld_mixed * 2, (uint64_t)(p.n * p.ld_mixed) * 2};
    const uint32_t box[4] = {64, 1, kC, 1};
    return sm100::encode_tensor_map(m, ptr, 4, dims, strides, box, B200_BF16, CU_TENSOR_MAP_L2_PROMOTION_L2_256B);
  };
  int st = map(&mq, mixed, p.dim, p.kv_heads);
  if (st == B200_OK) st = map(&mk, mixed + p.off_k, p.dim, p.kv_heads);
  if (st == B200_OK) st = map(&mv, mixed + p.off_v, p.vdim, p.heads);
  if (st != B200_OK) return st;
  delta_chunk_scan<DIM, VC, CW><<<(unsigned)(p.B * p.heads * vblocks), M::THREADS, M::BYTES, stream>>>(mq, mk, mv, p, n_chunks, vblocks);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

template <int DIM>
int launch_sized(const b200_delta_args& p, cudaStream_t stream) {
  int st = B200_ERR_UNSUPPORTED;
  switch (p.taps) {
    case 1: st = launch_conv<1>(p, stream); break;
    case 2: st = launch_conv<2>(p, stream); break;
    case 3: st = launch_conv<3>(p, stream); break;
    case 4: st = launch_conv<4>(p, stream); break;
    case 5: st = launch_conv<5>(p, stream); break;
    case 6: st = launch_conv<6>(p, stream); break;
    case 7: st = launch_conv<7>(p, stream); break;
    case 8: st = launch_conv<8>(p, stream); break;
  }
  if (st != B200_OK) return st;
  const int n_chunks = (int)((p.n + kC - 1) / kC);
  static std::atomic<bool> done[kMaxDevices];
  if (!opt_in(delta_chunk_prepare<DIM>, PrepareSmem<DIM>::BYTES, done)) return B200_ERR_CUDA;
  delta_chunk_prepare<DIM><<<(unsigned)(p.B * p.heads * n_chunks), 128, PrepareSmem<DIM>::BYTES, stream>>>(p, n_chunks);
  note_launches(1);
  // the widest column block that still gives every SM one
  const int64_t heads = p.B * p.heads;
  if (heads * ((p.vdim + 63) / 64) >= sm_count()) st = launch_scan<DIM, 64, 32>(p, n_chunks, stream);
  else if (heads * ((p.vdim + 31) / 32) >= sm_count()) st = launch_scan<DIM, 32, 16>(p, n_chunks, stream);
  else st = launch_scan<DIM, 16, 16>(p, n_chunks, stream);
  if (st != B200_OK) return st;
  return launch_finish(p, stream);
}

}  // namespace

bool delta_chunk_takes(const b200_delta_args& p) {
  return p.dtype == B200_BF16 && !p.pos_dev && p.n >= kC / 2 && p.dim <= 128 && p.vdim <= 512 && p.dim % 8 == 0 && p.vdim % 8 == 0 && p.taps <= 8 &&
         p.off_k % 8 == 0 && p.off_v % 8 == 0 && p.off_g % 8 == 0 && p.ld % 8 == 0 && p.ld_mixed % 8 == 0 && p.ld_y % 8 == 0 && p.conv_cols % 8 == 0 &&
         ((reinterpret_cast<uintptr_t>(p.rows) | reinterpret_cast<uintptr_t>(p.mixed) | reinterpret_cast<uintptr_t>(p.y) | reinterpret_cast<uintptr_t>(p.norm_w) |
           reinterpret_cast<uintptr_t>(p.state) | reinterpret_cast<uintptr_t>(p.conv_state) | reinterpret_cast<uintptr_t>(p.conv_w)) & 15) == 0 &&
         p.B <= 65535 && p.n <= 65535LL * kConvTokens && p.B * p.heads * p.n <= 0x7fffffffLL - 4096;
}

int64_t delta_chunk_workspace_bytes(const b200_delta_args& p) { return p.B * p.heads * ((p.n + kC - 1) / kC) * kRecordBytes; }

int launch_delta_chunk(const b200_delta_args& p, cudaStream_t stream) { return p.dim <= 64 ? launch_sized<64>(p, stream) : launch_sized<128>(p, stream); }

}  // namespace b200
