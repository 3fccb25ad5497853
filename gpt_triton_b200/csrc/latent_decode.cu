// One-token latent attention on tensor cores (bf16): the heads of a sequence share its cached latents, so a block takes
// 16 or 32 heads of one sequence and streams the latents once.
//   head_product_kernel   q~ = W_uk[head]^T q  before, and  W_uv[head] o~  after: one small product per head
//   latent_stream_kernel  scores q~ . c, online softmax and the weighted latent sum o~ over a range of the window
//   latent_merge_kernel   merges the ranges of one (sequence, head), adds the sink's term, normalises
// q~ is the output of a product, in bf16 like every other; the softmax weights are fp32 by definition and enter their MMA
// as two bf16 parts.
#include <atomic>

#include "mma_sync.cuh"

namespace b200 {
namespace {

using namespace warp_mma;

// ------------------------------------------------------------------ one product per head
// out[b, h, n] = sum_k a[b, h, k] * w[h, n, k] (K_MAJOR) or w[h, k, n].  Tile: 16 * MB sequences x 64 columns; MB = 1: the
// four warps take 16 columns each, MB = 4: 16 sequences each.  k, n multiples of 8.
template <bool K_MAJOR, int MB>
__global__ void __launch_bounds__(128)
head_product_kernel(const __nv_bfloat16* __restrict__ a, int64_t lda, int64_t a_head, const __nv_bfloat16* __restrict__ w, int64_t w_head, int64_t ldw,
                    __nv_bfloat16* __restrict__ out, int64_t ld_out, int64_t out_head, int B, int N, int K) {
  constexpr int ROWS = 16 * MB, NT = MB == 1 ? 2 : 8, STAGES = MB == 1 ? 4 : 3;
  __shared__ __align__(128) uint8_t tiles[STAGES][(ROWS + 64) * 128];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
  const int n0 = blockIdx.x * 64, h = blockIdx.y, b0 = blockIdx.z * ROWS;
  const int row_w = MB == 1 ? 0 : warp * 16, col_w = MB == 1 ? warp * 16 : 0;
  a += h * a_head, w += h * w_head, out += h * out_head;
  auto load = [&](int k0, int stage) {
    const uint32_t sa = (uint32_t)__cvta_generic_to_shared(tiles[stage]), sw = sa + ROWS * 128;
    for (int i = threadIdx.x; i < ROWS * 8; i += 128) {
      const int r = i >> 3, c = i & 7;
      const bool ok = b0 + r < B && k0 + c * 8 < K;
      cp_async16(sa + swz<128>(r, c), ok ? a + (int64_t)(b0 + r) * lda + k0 + c * 8 : a, ok);
    }
    for (int i = threadIdx.x; i < 64 * 8; i += 128) {
      const int r = i >> 3, c = i & 7;
      const int n = n0 + (K_MAJOR ? r : c * 8), k = k0 + (K_MAJOR ? c * 8 : r);
      const bool ok = n < N && k < K;
      cp_async16(sw + swz<128>(r, c), ok ? w + (K_MAJOR ? (int64_t)n * ldw + k : (int64_t)k * ldw + n) : w, ok);
    }
    cp_async_commit();
  };
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int i = 0; i < STAGES - 1; ++i) {
    if (i * 64 < K) load(i * 64, i);
    else cp_async_commit();  // (one group per step, so that the wait below can count them)
  }
  int stage = 0;
  for (int k0 = 0; k0 < K; k0 += 64) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();  // this step's tiles are in place, and the stage filled next is no longer read
    if (k0 + (STAGES - 1) * 64 < K) load(k0 + (STAGES - 1) * 64, stage == 0 ? STAGES - 1 : stage - 1);
    else cp_async_commit();
    const uint32_t sa = (uint32_t)__cvta_generic_to_shared(tiles[stage]), sw = sa + ROWS * 128;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t af[4];
      ldsm4(af, sa + swz<128>(row_w + (lane & 15), ks * 2 + (lane >> 4)));
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        uint32_t wf[4];
        const int n = col_w + np * 16;
        if (K_MAJOR) ldsm4(wf, sw + swz<128>(n + (lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1)));
        else ldsm4_trans(wf, sw + swz<128>(ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, n / 8 + (lane >> 4)));
        mma_bf16(acc[2 * np], af, wf[0], wf[1]);
        mma_bf16(acc[2 * np + 1], af, wf[2], wf[3]);
      }
    }
    if (++stage == STAGES) stage = 0;
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int b = b0 + row_w + g8 + r * 8, n = n0 + col_w + nt * 8 + t4 * 2;
      if (b < B && n < N) {
        *reinterpret_cast<__nv_bfloat162*>(out + (int64_t)b * ld_out + n) = __floats2bfloat162_rn(acc[nt][2 * r], acc[nt][2 * r + 1]);
      }
    }
}

// ------------------------------------------------------------------ streaming the latents
constexpr int kKeys = 32, kStreamThreads = 256;
constexpr int kPartRow = kKeys + 8;  // floats per row of partial scores (the padding spreads eight rows over the banks)

template <int RP, int HT>  // latent size, padded to 128, 256 or 512; 16-head tiles per block
struct StreamSmem {
  static constexpr int HEADS = 16 * HT;
  static constexpr int ROW = RP * 2;
  static constexpr int C_BYTES = kKeys * ROW;
  static constexpr int P_BYTES = HEADS * 128;  // one bf16 part of the weights; rows of 128 bytes, kKeys * 2 of them used
  static constexpr int S_BYTES = kStreamThreads / 32 * HEADS * kPartRow * 4;  // scores, one partial sum per eighth of the latent
  static constexpr int CTAS_PER_SM = HT == 1 ? 2 : 1;  // (the output of 32 heads takes too many registers for two)
  static constexpr int FIT = (220 * 1024 / CTAS_PER_SM - 2 * P_BYTES - S_BYTES) / C_BYTES;
  static constexpr int STAGES = FIT < 8 ? FIT : 8;  // tiles in the ring
  static constexpr int BYTES = STAGES * C_BYTES + 2 * P_BYTES + S_BYTES;
  static_assert(STAGES >= 2, "shared memory budget");
};

// Per tile of 32 latents: partial scores (a warp takes all keys over an eighth of the latent; its part of q~ stays in
// registers), softmax (a warp takes whole heads, one key per lane), weighted sum (a warp takes an eighth of the latent),
// with a barrier in front of each.
// blockIdx.x = sequence, y = group of 16 * HT heads, z = range of the window.  Partial results per (sequence, head, range):
// part_ml = (maximum in log2 units, denominator), part_o = unnormalised sum of latents.
// Shared-memory addresses of the weighted sum: a row's 16-byte pieces are permuted inside groups of eight by the row's low three bits, so a
// lane's address of piece 2 i + b is one of four precomputed offsets (i mod 4) plus 128 bytes for every further four.
template <int RP, int HT>
__global__ void __launch_bounds__(kStreamThreads, StreamSmem<RP, HT>::CTAS_PER_SM)
latent_stream_kernel(const __nv_bfloat16* __restrict__ qt, const __nv_bfloat16* __restrict__ cache, float* __restrict__ part_o, float2* __restrict__ part_ml,
                     int heads, int R, int64_t ring, int64_t window, float scale_log2e, const int* __restrict__ pos_dev) {
  using M = StreamSmem<RP, HT>;
  constexpr int WARPS = kStreamThreads / 32, HEADS = M::HEADS;
  constexpr int ROW = M::ROW, NT = RP / 8 / WARPS;  // 8-column output tiles per warp
  constexpr int PIECES = RP / 8, ROWS_PER_PASS = kStreamThreads / PIECES, PASSES = kKeys / ROWS_PER_PASS;
  static_assert(kStreamThreads % PIECES == 0 && kKeys % ROWS_PER_PASS == 0, "a thread keeps its column of pieces");
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float s_mult[HEADS];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
  const int64_t b = blockIdx.x;
  const int h0 = blockIdx.y * HEADS, split = blockIdx.z, n_split = gridDim.z;
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem);
  const uint32_t p_hi = base + M::STAGES * M::C_BYTES, p_lo = p_hi + M::P_BYTES;
  float* s_part = reinterpret_cast<float*>(smem + M::STAGES * M::C_BYTES + 2 * M::P_BYTES);  // [WARPS][HEADS][kPartRow]
  const int64_t pos = pos_dev[0], first = pos + 1 > window ? pos + 1 - window : 0;
  const int n_keys = pos < 0 ? 0 : (int)(pos - first + 1);
  const int tiles = (n_keys + kKeys - 1) / kKeys, per = (tiles + n_split - 1) / n_split;
  const int tile0 = split * per, tile1 = min(tiles, tile0 + per);

  const __nv_bfloat16* cb = cache + b * ring * R;
  const int slot0 = (int)(first % ring), n_ring = (int)ring;
  // this thread's 16-byte pieces of a tile: always column ld_c, rows ld_r, ld_r + ROWS_PER_PASS, ...
  const int ld_c = threadIdx.x % PIECES, ld_r = threadIdx.x / PIECES;
  const bool col_ok = ld_c * 8 < R;
  const __nv_bfloat16* ld_src = cb + ld_c * 8;
  auto load = [&](int tile, int stage) {
    const uint32_t dst = base + stage * M::C_BYTES;
    const int key0 = tile * kKeys + ld_r;
#pragma unroll
    for (int i = 0; i < PASSES; ++i) {
      const int key = key0 + i * ROWS_PER_PASS;
      int slot = slot0 + key;  // (key < window <= ring: one wrap at most)
      if (slot >= n_ring) slot -= n_ring;
      const bool ok = key < n_keys && col_ok;
      cp_async16(dst + swz<ROW>(ld_r + i * ROWS_PER_PASS, ld_c), ok ? ld_src + (int64_t)slot * R : cb, ok);
    }
    cp_async_commit();
  };
  // this warp's eighth of the queries as A fragments (rows g8, g8 + 8; columns t4 * 2 + {0, 1} and + 8 of each 16)
  constexpr int KS = RP / 8 / WARPS / 2;  // 16-wide k-steps per warp
  uint32_t qf[HT][KS][4];
#pragma unroll
  for (int ht = 0; ht < HT; ++ht)
#pragma unroll
    for (int ks = 0; ks < KS; ++ks)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = h0 + ht * 16 + g8 + (e & 1) * 8, c = (warp * KS + ks) * 16 + t4 * 2 + (e >> 1) * 8;
        qf[ht][ks][e] = h < heads && c < R ? *reinterpret_cast<const uint32_t*>(qt + (b * heads + h) * R + c) : 0u;
      }
  uint32_t off_c[KS], off_v[4];  // lane addresses: scores, by k-step; weighted sum, of piece 2 i + b, i mod 4
#pragma unroll
  for (int i = 0; i < KS; ++i) off_c[i] = swz<ROW>((lane & 7) + ((lane >> 4) << 3), (warp * KS + i) * 2 + ((lane >> 3) & 1));
#pragma unroll
  for (int i = 0; i < 4; ++i)
    off_v[i] = swz<ROW>((lane & 7) + ((lane >> 3) & 1) * 8, (warp * NT + i * 2 + (lane >> 4)) & 7) + (uint32_t)((warp * NT / 8) * 128);
  constexpr int V_WRAP = NT >= 8 ? 4 : NT / 2;  // pairs of output tiles before a warp's pieces enter the next group of eight

  float o[HT][NT][4];
#pragma unroll
  for (int ht = 0; ht < HT; ++ht)
#pragma unroll
    for (int i = 0; i < NT; ++i) o[ht][i][0] = o[ht][i][1] = o[ht][i][2] = o[ht][i][3] = 0.f;
  constexpr int HPW = HEADS / WARPS;  // heads whose softmax this warp keeps
  float m_run[HPW], l_run[HPW];
#pragma unroll
  for (int i = 0; i < HPW; ++i) m_run[i] = -INFINITY, l_run[i] = 0.f;
#pragma unroll
  for (int i = 0; i < M::STAGES - 1; ++i) {
    if (tile0 + i < tile1) load(tile0 + i, i);
    else cp_async_commit();  // (one group per tile, so that the wait below can count them)
  }
  int stage = 0;
  for (int tile = tile0; tile < tile1; ++tile, stage = stage + 1 == M::STAGES ? 0 : stage + 1) {
    cp_async_wait<M::STAGES - 2>();
    __syncthreads();  // the tile has landed; the stage before it and the weights of the tile before are no longer read
    if (tile + M::STAGES - 1 < tile1) load(tile + M::STAGES - 1, stage == 0 ? M::STAGES - 1 : stage - 1);
    else cp_async_commit();
    const uint32_t sc = base + stage * M::C_BYTES;
    {
      float s[HT][kKeys / 8][4];
#pragma unroll
      for (int ht = 0; ht < HT; ++ht)
#pragma unroll
        for (int nt = 0; nt < kKeys / 8; ++nt) s[ht][nt][0] = s[ht][nt][1] = s[ht][nt][2] = s[ht][nt][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks)
#pragma unroll
        for (int np = 0; np < kKeys / 16; ++np) {
          uint32_t cf[4];
          ldsm4(cf, sc + off_c[ks] + np * 16 * ROW);
#pragma unroll
          for (int ht = 0; ht < HT; ++ht) {
            mma_bf16(s[ht][2 * np], qf[ht][ks], cf[0], cf[1]);
            mma_bf16(s[ht][2 * np + 1], qf[ht][ks], cf[2], cf[3]);
          }
        }
#pragma unroll
      for (int ht = 0; ht < HT; ++ht)
#pragma unroll
        for (int nt = 0; nt < kKeys / 8; ++nt)
#pragma unroll
          for (int r = 0; r < 2; ++r)
            *reinterpret_cast<float2*>(s_part + (warp * HEADS + ht * 16 + g8 + r * 8) * kPartRow + nt * 8 + t4 * 2) =
                make_float2(s[ht][nt][2 * r], s[ht][nt][2 * r + 1]);
    }
    __syncthreads();
    const bool key_ok = tile * kKeys + lane < n_keys;
#pragma unroll
    for (int i = 0; i < HPW; ++i) {
      const int row = warp * HPW + i;
      float v = 0.f;
#pragma unroll
      for (int w2 = 0; w2 < WARPS; ++w2) v += s_part[(w2 * HEADS + row) * kPartRow + lane];
      v = key_ok ? v * scale_log2e : -INFINITY;
      float m_new = v;
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) m_new = fmaxf(m_new, __shfl_xor_sync(0xffffffffu, m_new, off));
      m_new = fmaxf(m_run[i], m_new);  // finite: a tile has at least one key
      const float mult = exp2f(m_run[i] - m_new), p = exp2f(v - m_new);
      m_run[i] = m_new;
      l_run[i] = l_run[i] * mult + warp_sum(p);
      const __nv_bfloat16 hi = __float2bfloat16_rn(p), lo = __float2bfloat16_rn(p - __bfloat162float(hi));
      const uint32_t at = swz<128>(row, lane >> 3) + (lane & 7) * 2;
      asm volatile("st.shared.b16 [%0], %1;" ::"r"(p_hi + at), "h"(*reinterpret_cast<const uint16_t*>(&hi)) : "memory");
      asm volatile("st.shared.b16 [%0], %1;" ::"r"(p_lo + at), "h"(*reinterpret_cast<const uint16_t*>(&lo)) : "memory");
      if (lane == 0) s_mult[row] = mult;
    }
    __syncthreads();
    float mult[HT][2];
    bool moved = false;
#pragma unroll
    for (int ht = 0; ht < HT; ++ht)
#pragma unroll
      for (int r = 0; r < 2; ++r) mult[ht][r] = s_mult[ht * 16 + g8 + r * 8], moved |= mult[ht][r] != 1.0f;
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int ht = 0; ht < HT; ++ht)
#pragma unroll
        for (int i = 0; i < NT; ++i)
          o[ht][i][0] *= mult[ht][0], o[ht][i][1] *= mult[ht][0], o[ht][i][2] *= mult[ht][1], o[ht][i][3] *= mult[ht][1];
    }
    // o~ += P c for this warp's RP / WARPS columns
#pragma unroll
    for (int kk = 0; kk < kKeys / 16; ++kk) {
      uint32_t ph[HT][4], pl[HT][4];
#pragma unroll
      for (int ht = 0; ht < HT; ++ht) {
        const uint32_t at = swz<128>(ht * 16 + (lane & 15), kk * 2 + (lane >> 4));
        ldsm4(ph[ht], p_hi + at);
        ldsm4(pl[ht], p_lo + at);
      }
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        uint32_t cf[4];
        ldsm4_trans(cf, sc + off_v[np % V_WRAP] + (np / V_WRAP) * 128 + kk * 16 * ROW);
#pragma unroll
        for (int ht = 0; ht < HT; ++ht) {
          mma_bf16(o[ht][2 * np], ph[ht], cf[0], cf[1]);
          mma_bf16(o[ht][2 * np + 1], ph[ht], cf[2], cf[3]);
          mma_bf16(o[ht][2 * np], pl[ht], cf[0], cf[1]);
          mma_bf16(o[ht][2 * np + 1], pl[ht], cf[2], cf[3]);
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    const int h = h0 + warp * HPW + i;
    if (lane == 0 && h < heads) part_ml[(b * heads + h) * n_split + split] = make_float2(m_run[i], l_run[i]);
  }
#pragma unroll
  for (int ht = 0; ht < HT; ++ht)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int h = h0 + ht * 16 + g8 + r * 8;
      if (h >= heads) continue;
      const int64_t item = (b * heads + h) * n_split + split;
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int c = (warp * NT + i) * 8 + t4 * 2;
        if (c < R) *reinterpret_cast<float2*>(part_o + item * R + c) = make_float2(o[ht][i][2 * r], o[ht][i][2 * r + 1]);
      }
    }
}

// One block per (sequence, head).
constexpr int kMaxSplit = 64;
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part_o, const float2* __restrict__ part_ml, __nv_bfloat16* __restrict__ ot, int heads, int R, int n_split,
                    const float* __restrict__ sink) {
  __shared__ float factor[kMaxSplit];
  const int64_t item = blockIdx.x;
  const int h = (int)(item % heads), lane = threadIdx.x & 31;
  if (threadIdx.x < 32) {
    float2 ml[kMaxSplit / 32];
    float m = -INFINITY, l = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxSplit / 32; ++i) {
      const int s = i * 32 + lane;
      ml[i] = s < n_split ? part_ml[item * n_split + s] : make_float2(-INFINITY, 0.f);
      m = fmaxf(m, ml[i].x);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
#pragma unroll
    for (int i = 0; i < kMaxSplit / 32; ++i) l = fmaf(ml[i].y, exp2f(ml[i].x - m), l);
    l = warp_sum(l);
    if (sink) l += exp2f(sink[h] * 1.4426950408889634f - m);
    const float inv = 1.0f / l;
#pragma unroll
    for (int i = 0; i < kMaxSplit / 32; ++i) factor[i * 32 + lane] = exp2f(ml[i].x - m) * inv;
  }
  __syncthreads();
  for (int r = threadIdx.x * 4; r < R; r += 512) {  // (R is a multiple of 8)
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < n_split; ++s) {
      const float f = factor[s];
      const float4 o = *reinterpret_cast<const float4*>(part_o + (item * n_split + s) * R + r);
      v.x = fmaf(o.x, f, v.x), v.y = fmaf(o.y, f, v.y), v.z = fmaf(o.z, f, v.z), v.w = fmaf(o.w, f, v.w);
    }
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(ot + item * R + r) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
  }
}

size_t round256(size_t v) { return (v + 255) & ~(size_t)255; }

struct Plan {
  int n_split;
  size_t off_po, off_ml, off_ot, bytes;
};
Plan make_plan(int64_t B, int64_t heads, int64_t R, int64_t window) {
  Plan p;
  const int64_t per_block = heads > 16 ? 32 : 16, groups = B * ((heads + per_block - 1) / per_block), tiles = (window + kKeys - 1) / kKeys;
  // ranges per sequence: the fewest rounds of blocks, counted in tiles (a block's start-up and its share of the merge are
  // worth about three)
  const int64_t slots = (int64_t)sm_count() * (heads > 16 ? 1 : 2);
  int64_t n = 1, best = -1;
  for (int64_t k = 1; k <= tiles && k <= kMaxSplit; ++k) {
    const int64_t cost = ((groups * k + slots - 1) / slots) * ((tiles + k - 1) / k + 3);
    if (best < 0 || cost < best) best = cost, n = k;
  }
  p.n_split = (int)n;
  size_t at = round256((size_t)(B * heads * R) * 2);  // q~
  p.off_po = at, at += round256((size_t)(B * heads * n * R) * 4);
  p.off_ml = at, at += round256((size_t)(B * heads * n) * 8);
  p.off_ot = at, at += round256((size_t)(B * heads * R) * 2);
  p.bytes = at;
  return p;
}

template <int RP, int HT>
int launch_stream(const __nv_bfloat16* qt, const void* cache, float* po, float2* ml, int64_t B, int64_t heads, int64_t R, int64_t ring, int64_t window,
                  float scale, int n_split, const int* pos_dev, cudaStream_t stream) {
  constexpr int smem = StreamSmem<RP, HT>::BYTES;
  static std::atomic<bool> attr_set[kMaxDevices];
  const int slot = device_slot();
  if (slot < 0) return B200_ERR_CUDA;
  if (!attr_set[slot].load(std::memory_order_acquire)) {
    if (cudaFuncSetAttribute(latent_stream_kernel<RP, HT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return B200_ERR_CUDA;
    attr_set[slot].store(true, std::memory_order_release);
  }
  latent_stream_kernel<RP, HT><<<dim3((unsigned)B, (unsigned)((heads + 16 * HT - 1) / (16 * HT)), (unsigned)n_split), kStreamThreads, smem, stream>>>(
      qt, static_cast<const __nv_bfloat16*>(cache), po, ml, (int)heads, (int)R, ring, window, scale * 1.4426950408889634f, pos_dev);
  note_launches(1);
  return status_from_cuda(cudaGetLastError());
}

template <int RP>
int launch_stream_heads(const __nv_bfloat16* qt, const void* cache, float* po, float2* ml, int64_t B, int64_t heads, int64_t R, int64_t ring,
                        int64_t window, float scale, int n_split, const int* pos_dev, cudaStream_t stream) {
  return heads > 16 ? launch_stream<RP, 2>(qt, cache, po, ml, B, heads, R, ring, window, scale, n_split, pos_dev, stream)
                    : launch_stream<RP, 1>(qt, cache, po, ml, B, heads, R, ring, window, scale, n_split, pos_dev, stream);
}

template <bool K_MAJOR>
void head_product(const __nv_bfloat16* a, int64_t lda, int64_t a_head, const __nv_bfloat16* w, int64_t w_head, int64_t ldw, __nv_bfloat16* out, int64_t ld_out,
                  int64_t out_head, int64_t B, int64_t heads, int64_t N, int64_t K, cudaStream_t stream) {
  const unsigned nb = (unsigned)((N + 63) / 64);
  if (B <= 128)
    head_product_kernel<K_MAJOR, 1><<<dim3(nb, (unsigned)heads, (unsigned)((B + 15) / 16)), 128, 0, stream>>>(a, lda, a_head, w, w_head, ldw, out, ld_out, out_head, (int)B, (int)N, (int)K);
  else
    head_product_kernel<K_MAJOR, 4><<<dim3(nb, (unsigned)heads, (unsigned)((B + 63) / 64)), 128, 0, stream>>>(a, lda, a_head, w, w_head, ldw, out, ld_out,
                                                                                                                    out_head, (int)B, (int)N, (int)K);
  note_launches(1);
}

bool aligned16_all(const void* a, const void* b, const void* c, const void* d) {
  return ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(c) | reinterpret_cast<uintptr_t>(d)) & 15) == 0;
}

}  // namespace

size_t latent_decode_mma_workspace_bytes(int64_t B, int64_t heads, int64_t R, int64_t window) { return make_plan(B, heads, R, window).bytes; }

int launch_latent_decode_mma(const void* q, int64_t ld_q, const void* w_uk, const void* w_uv, const void* cache, void* out, int64_t ld_out, int64_t B,
                             int64_t heads, int64_t dim, int64_t vdim, int64_t R, int64_t ring, int64_t window, float scale, const float* sink,
                             const int* pos_dev, void* workspace, cudaStream_t stream) {
  if (R > 512 || R % 8 || dim % 8 || vdim % 8 || ld_q % 8 || ld_out % 2 || (reinterpret_cast<uintptr_t>(out) & 3) || !aligned16_all(q, w_uk, w_uv, cache)) return B200_ERR_UNSUPPORTED;
  if (B > 65535 || heads > 65535 || ring > (1 << 30)) return B200_ERR_UNSUPPORTED;
  const Plan p = make_plan(B, heads, R, window);
  uint8_t* ws = static_cast<uint8_t*>(workspace);
  __nv_bfloat16* qt = reinterpret_cast<__nv_bfloat16*>(ws);
  float* po = reinterpret_cast<float*>(ws + p.off_po);
  float2* ml = reinterpret_cast<float2*>(ws + p.off_ml);
  __nv_bfloat16* ot = reinterpret_cast<__nv_bfloat16*>(ws + p.off_ot);
  head_product<false>((const __nv_bfloat16*)q, ld_q, dim, (const __nv_bfloat16*)w_uk, dim * R, R, qt, heads * R, R, B, heads, R, dim, stream);
  int st = R <= 128   ? launch_stream_heads<128>(qt, cache, po, ml, B, heads, R, ring, window, scale, p.n_split, pos_dev, stream)
           : R <= 256 ? launch_stream_heads<256>(qt, cache, po, ml, B, heads, R, ring, window, scale, p.n_split, pos_dev, stream)
                      : launch_stream_heads<512>(qt, cache, po, ml, B, heads, R, ring, window, scale, p.n_split, pos_dev, stream);
  if (st != B200_OK) return st;
  latent_merge_kernel<<<(unsigned)(B * heads), 128, 0, stream>>>(po, ml, ot, (int)heads, (int)R, p.n_split, sink);
  note_launches(1);
  head_product<true>(ot, heads * R, R, (const __nv_bfloat16*)w_uv, vdim * R, R, (__nv_bfloat16*)out, ld_out, vdim, B, heads, vdim, R, stream);
  return status_from_cuda(cudaGetLastError());
}

}  // namespace b200
