// Differential attention over a prompt on the 5th-generation tensor cores (bf16 queries and keys, fp16 values; sizes up to
// 64 or 128, smaller ones zero-filled by the loads): sliding window, grouped key/value heads, soft-capped scores.
//
// Work item = up to 128 query rows of one (sequence, head), BOTH maps, so that a block of values is loaded once for the two
// and their difference, its norm and the gate are finished where the accumulators are.  Persistent CTAs, one per SM:
//   warp 0       TMA producer: the two query tiles (buffered while the item before is computed) and, per 64-key block, two
//                key tiles and one value tile
//   warp 1       tcgen05.mma issuer: S_m = Q_m K_m^T (tensor memory, double-buffered per map, issued one block ahead) and
//                O_m (+)= P_m V
//   warps 2-9    softmax of map 0, warps 10-17 of map 1, two threads per query row each, as in attention_sm100.cu; the two
//                maps' chains (scores -> cap -> maximum -> exponentials -> P) run side by side
// At the end of an item the four threads of a row exchange the denominators, take a quarter of the columns each of
// o = O_0 / l_0 - lambda O_1 / l_1, exchange their sums of squares and store o * (norm, scale, gate).
// The cap cap * tanh(s / cap) must be as exact as fp32 scores are (tanh.approx is not): an odd polynomial (error 1e-8) while
// every |s / cap| of a warp is below 0.75, else 1 - 2 / (1 + exp(2 s / cap)).
#include <atomic>

#include "attention_sm100.cuh"

namespace b200 {
namespace pair100 {

using namespace attn100;

constexpr int SOFTMAX_WARPS = 8;  // per map
constexpr int FIRST_SOFTMAX = 2;
constexpr int THREADS = 32 * (FIRST_SOFTMAX + 2 * SOFTMAX_WARPS);
constexpr int P_BYTES = BLOCK_M * BLOCK_N * 2;
constexpr int CTRL = 512;
constexpr int XCHG_FLOATS = 2 * 2 * 2 * BLOCK_M + 2 * 2 * BLOCK_M + 2 * 2 * BLOCK_M;  // block maxima [map][slot][half], denominators and squares [map][half]
constexpr int TMEM = 512;         // S[map][2] (64 columns each) + O[map]

template <int KD, int VD>
struct Shape {
  static constexpr int KA = KD / 64, VA = VD / 64;  // atoms of 64 columns (128 bytes)
  static constexpr int Q_BUFS = KD == 64 ? 2 : 1;
  static constexpr int STAGES = KD == 64 ? 3 : 2;
  static constexpr int Q_ATOM = BLOCK_M * 128, KV_ATOM = BLOCK_N * 128;
  static constexpr int Q_MAP = KA * Q_ATOM, Q_BYTES = 2 * Q_MAP;
  static constexpr int K_MAP = KA * KV_ATOM, V_AT = 2 * K_MAP, STAGE = V_AT + VA * KV_ATOM;
  static constexpr int SMEM = Q_BUFS * Q_BYTES + STAGES * STAGE + 2 * P_BYTES + 1024 + CTRL + XCHG_FLOATS * 4;
  static_assert(SMEM <= 227 * 1024, "shared memory budget");
  static_assert(4 * BLOCK_N + 2 * VD <= TMEM, "tensor memory budget");
};

struct Args {
  __nv_bfloat16* out;
  int64_t ld_out;
  const __nv_bfloat16* gate;
  int64_t ld_gate;
  const float* lambda;
  int B, H, group, L, hist, window, vdim;  // group: query heads per key/value head
  float scale_log2e, to_z, cap_log2e;      // softcap: z = s * to_z, score (log2 units) = cap_log2e * tanh(z); cap_log2e = 0: score = s * scale_log2e
  float eps, out_scale;
  int q_head_inner, k_head_inner, v_head_inner;
  int* status_word;
};

struct Work {
  int b, h, q0, q_end, k0, nblk;
};
__device__ __forceinline__ Work decode_work(int64_t idx, int bh, int n_qt, const Args& p) {
  const int qt = n_qt - 1 - (int)(idx / bh), r = (int)(idx % bh);
  Work w;
  w.b = r / p.H;
  w.h = r % p.H;
  w.q0 = qt == 0 ? 0 : tile_end(qt - 1, n_qt, p.L);
  w.q_end = tile_end(qt, n_qt, p.L);
  w.k0 = max(0, p.hist + w.q0 - p.window + 1);
  w.nblk = (p.hist + w.q_end - w.k0 + BLOCK_N - 1) / BLOCK_N;
  return w;
}

// cap_log2e * tanh(z) for |z| < 0.75, two at a time
__device__ __forceinline__ float2 cap_small(float2 s, float to_z, float cap) {
  const float2 z = __fmul2_rn(s, make_float2(to_z, to_z)), w = __fmul2_rn(z, z);
  auto k = [](float c) { return make_float2(c, c); };
  float2 p = __ffma2_rn(w, k(-4.500336705e-03f), k(1.924961053e-02f));
  p = __ffma2_rn(w, p, k(-5.315760410e-02f));
  p = __ffma2_rn(w, p, k(1.332083726e-01f));
  p = __ffma2_rn(w, p, k(-3.333250593e-01f));
  p = __ffma2_rn(w, p, k(9.999998481e-01f));
  return __fmul2_rn(__fmul2_rn(z, make_float2(cap, cap)), p);
}
__device__ __forceinline__ float cap_any(float s, float to_z, float cap) {
  const float e = ex2f(s * to_z * 2.8853900817779268f);  // exp(2 z)
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
  return fmaf(-2.0f * cap, r, cap);
}

__device__ __forceinline__ void tmem_ld_32x16(uint32_t taddr, uint32_t (&v)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]), "=r"(v[9]), "=r"(v[10]),
        "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
      : "r"(taddr));
}

template <int KD, int VD>
__global__ void __launch_bounds__(THREADS, 1)
pair_attention_sm100_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                            Args p, uint32_t idesc_s, uint32_t idesc_pv) {
  using C = Shape<KD, VD>;
  constexpr int STAGES = C::STAGES, Q_BUFS = C::Q_BUFS;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (base - raw);
  const uint32_t smem_q = base;                                 // [Q_BUFS][map]
  const uint32_t smem_kv = smem_q + Q_BUFS * C::Q_BYTES;        // [STAGES]{K_0, K_1, V}
  const uint32_t smem_p = smem_kv + STAGES * C::STAGE;          // [map][128][64] fp16
  uint8_t* ctrl = smem + Q_BUFS * C::Q_BYTES + STAGES * C::STAGE + 2 * P_BYTES;
  const uint32_t bars = smem_u32(ctrl);
  const uint32_t bar_q_full = bars;                             // [Q_BUFS]
  const uint32_t bar_q_empty = bar_q_full + 16;                 // [Q_BUFS]
  const uint32_t bar_kv_full = bar_q_empty + 16;                // [STAGES]
  const uint32_t bar_kv_empty = bar_kv_full + 8 * STAGES;       // [STAGES]
  const uint32_t bar_s_full = bar_kv_empty + 8 * STAGES;        // [map][2]
  const uint32_t bar_s_empty = bar_s_full + 32;                 // [map][2]
  const uint32_t bar_p_full = bar_s_empty + 32;                 // [map]
  const uint32_t bar_pv_done = bar_p_full + 16;                 // [map]
  const uint32_t bar_pair = bar_pv_done + 16;                   // [map][4]: the two warps of a map that share 32 rows
  const uint32_t bar_row = bar_pair + 64;                       // [4]: the four warps that share 32 rows
  constexpr int BAR_BYTES = 32 + 16 * STAGES + 64 + 32 + 64 + 32;
  static_assert(BAR_BYTES + 16 <= CTRL, "control block too small");
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(ctrl + BAR_BYTES);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(ctrl + BAR_BYTES + 8);
  float* xchg = reinterpret_cast<float*>(ctrl + CTRL);
  float* row_l = xchg + 8 * BLOCK_M;   // [map][half][128]
  float* row_sq = row_l + 4 * BLOCK_M;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_qt = (p.L + BLOCK_M - 1) / BLOCK_M;
  const int bh = p.B * p.H;
  const int64_t n_items = (int64_t)n_qt * bh;

  if (threadIdx.x == 0) {
    for (int i = 0; i < Q_BUFS; ++i) {
      mbar_init(bar_q_full + 8 * i, 1);
      mbar_init(bar_q_empty + 8 * i, 1);
    }
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(bar_kv_full + 8 * i, 1);
      mbar_init(bar_kv_empty + 8 * i, 1);
    }
    for (int i = 0; i < 4; ++i) {
      mbar_init(bar_s_full + 8 * i, 1);
      mbar_init(bar_s_empty + 8 * i, SOFTMAX_WARPS);
      mbar_init(bar_row + 8 * i, 4);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(bar_p_full + 8 * i, SOFTMAX_WARPS);
      mbar_init(bar_pv_done + 8 * i, 1);
    }
    for (int i = 0; i < 8; ++i) mbar_init(bar_pair + 8 * i, 2);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    fence_proxy_async_smem();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), TMEM);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t tmem_o = tmem_base + 4 * BLOCK_N;  // O[map]: VD columns each, behind S[map][2]

  if (warp == 0) {
    // ------------------------------------------------------------ TMA producer
    if (lane == 0) {
      uint32_t qi = 0, ki = 0;
      bool alive = true;
      for (int64_t idx = blockIdx.x; idx < n_items && alive; idx += gridDim.x) {
        const Work w = decode_work(idx, bh, n_qt, p);
        const int g = w.h / p.group;
        const uint32_t qb = qi % Q_BUFS;
        if (!mbar_wait(bar_q_empty + 8 * qb, ((qi / Q_BUFS) & 1) ^ 1u, abort_flag, p.status_word, 61)) break;
        mbar_arrive_expect_tx(bar_q_full + 8 * qb, C::Q_BYTES);
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int a = 0; a < C::KA; ++a)
            tma_load_4d(smem_q + qb * C::Q_BYTES + m * C::Q_MAP + a * C::Q_ATOM, &map_q, bar_q_full + 8 * qb, 64 * a, p.q_head_inner ? 2 * w.h + m : w.q0,
                        p.q_head_inner ? w.q0 : 2 * w.h + m, w.b);
        ++qi;
        for (int j = 0; j < w.nblk; ++j) {
          const uint32_t st = ki % STAGES;
          if (!mbar_wait(bar_kv_empty + 8 * st, ((ki / STAGES) & 1) ^ 1u, abort_flag, p.status_word, 62)) {
            alive = false;
            break;
          }
          mbar_arrive_expect_tx(bar_kv_full + 8 * st, C::STAGE);
          const int key = w.k0 + j * BLOCK_N;
          const uint32_t dst = smem_kv + st * C::STAGE;
#pragma unroll
          for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int a = 0; a < C::KA; ++a)
              tma_load_4d(dst + m * C::K_MAP + a * C::KV_ATOM, &map_k, bar_kv_full + 8 * st, 64 * a, p.k_head_inner ? 2 * g + m : key,
                          p.k_head_inner ? key : 2 * g + m, w.b);
#pragma unroll
          for (int a = 0; a < C::VA; ++a)
            tma_load_4d(dst + C::V_AT + a * C::KV_ATOM, &map_v, bar_kv_full + 8 * st, 64 * a, p.v_head_inner ? g : key, p.v_head_inner ? key : g, w.b);
          ++ki;
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      uint32_t qi = 0, ks = 0, kp = 0;  // items; key blocks whose scores / products have been issued
      bool alive = true;
      auto issue_s = [&](uint32_t qb) -> bool {
        const uint32_t st = ks % STAGES, sb = ks & 1;
        if (!mbar_wait(bar_kv_full + 8 * st, (ks / STAGES) & 1, abort_flag, p.status_word, 63)) return false;
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          if (!mbar_wait(bar_s_empty + 16 * m + 8 * sb, ((ks >> 1) & 1) ^ 1u, abort_flag, p.status_word, 64)) return false;
          tc_fence_after();
          const uint64_t da = desc_kmajor(smem_q + qb * C::Q_BYTES + m * C::Q_MAP);
          const uint64_t db = desc_kmajor(smem_kv + st * C::STAGE + m * C::K_MAP);
#pragma unroll
          for (int k = 0; k < KD / 16; ++k)
            umma_f16(tmem_base + (uint32_t)((2 * m + sb) * BLOCK_N), da + (uint64_t)(2 * (k & 3) + (k >> 2) * (C::Q_ATOM >> 4)),
                     db + (uint64_t)(2 * (k & 3) + (k >> 2) * (C::KV_ATOM >> 4)), idesc_s, (uint32_t)(k != 0));
          umma_commit(bar_s_full + 16 * m + 8 * sb);
        }
        ++ks;
        return true;
      };
      for (int64_t idx = blockIdx.x; idx < n_items && alive; idx += gridDim.x) {
        const Work w = decode_work(idx, bh, n_qt, p);
        const uint32_t qb = qi % Q_BUFS;
        if (!mbar_wait(bar_q_full + 8 * qb, (qi / Q_BUFS) & 1, abort_flag, p.status_word, 65)) break;
        if (!issue_s(qb)) break;
        for (int j = 0; j < w.nblk && alive; ++j) {
          if (j + 1 < w.nblk) {
            if (!issue_s(qb)) {
              alive = false;
              break;
            }
          } else {
            umma_commit(bar_q_empty + 8 * qb);  // every S of this item is issued: Q is free once they finish
          }
          const uint32_t st = kp % STAGES;
          const uint64_t db = desc_mnmajor(smem_kv + st * C::STAGE + C::V_AT, C::VA == 1 ? 1024 : C::KV_ATOM);
#pragma unroll
          for (int m = 0; m < 2; ++m) {
            if (!mbar_wait(bar_p_full + 8 * m, kp & 1, abort_flag, p.status_word, 66)) {
              alive = false;
              break;
            }
            tc_fence_after();
            const uint64_t da = desc_kmajor(smem_p + m * P_BYTES);
#pragma unroll
            for (int k = 0; k < BLOCK_N / 16; ++k)
              umma_f16(tmem_o + (uint32_t)(m * VD), da + (uint64_t)(2 * k), db + (uint64_t)(128 * k), idesc_pv, (uint32_t)((j | k) != 0));
            umma_commit(bar_pv_done + 8 * m);
          }
          if (!alive) break;
          umma_commit(bar_kv_empty + 8 * st);
          ++kp;
        }
        ++qi;
      }
    }
  } else {
    // ------------------------------------------------------------ softmax warps
    const int map = (warp - FIRST_SOFTMAX) >> 3, half = ((warp - FIRST_SOFTMAX) >> 2) & 1;
    const int quarter = warp & 3;  // tensor-memory lanes [32 * quarter, +32)
    const int r_in_tile = quarter * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(quarter * 32) << 16;
    const uint32_t p_row = smem_p + (uint32_t)map * P_BYTES + (uint32_t)r_in_tile * 128u;
    const uint32_t sw = (uint32_t)(r_in_tile & 7);
    const uint32_t s_addr = tmem_base + lane_addr + (uint32_t)(2 * map * BLOCK_N + half * 32);
    const uint32_t o_addr = tmem_o + lane_addr + (uint32_t)(map * VD + half * (VD / 2));
    float* my_x = xchg + (map * 4 + half) * BLOCK_M + r_in_tile;  // slot s: + s * 2 * BLOCK_M
    const float* partner_x = xchg + (map * 4 + (half ^ 1)) * BLOCK_M + r_in_tile;
    const uint32_t my_pair_bar = bar_pair + 8 * (uint32_t)(map * 4 + quarter);
    const uint32_t my_row_bar = bar_row + 8 * (uint32_t)quarter;
    uint32_t xphase = 0, rphase = 0;
    // the four warps of a row quarter have arrived (false: the CTA is aborting)
    auto meet = [&]() -> bool {
      __syncwarp();
      if (lane == 0) mbar_arrive(my_row_bar);
      if (!mbar_wait(my_row_bar, rphase, abort_flag, p.status_word, 72)) return false;
      rphase ^= 1u;
      return true;
    };
    const float lambda = __ldg(p.lambda);
    const bool capped = p.cap_log2e > 0.f;
    const float small_s = capped ? 0.75f / p.to_z : 0.f;  // |s| below this: the polynomial
    uint32_t it_count = 0;
    bool alive = true;
    for (int64_t idx = blockIdx.x; idx < n_items && alive; idx += gridDim.x) {
      const Work w = decode_work(idx, bh, n_qt, p);
      const int row = w.q0 + r_in_tile;
      const int krow = row + p.hist, warp_krow0 = w.q0 + quarter * 32 + p.hist;
      const bool warp_live = w.q0 + quarter * 32 < w.q_end;
      float m_run = -INFINITY, l_run = 0.f;
      for (int j = 0; j < w.nblk; ++j, ++it_count) {
        const uint32_t sb = it_count & 1;
        if (!mbar_wait(bar_s_full + 16 * map + 8 * sb, (it_count >> 1) & 1, abort_flag, p.status_word, 67)) {
          alive = false;
          break;
        }
        tc_fence_after();
        const int k0 = w.k0 + j * BLOCK_N + half * 32;
        const bool live = warp_live && k0 <= warp_krow0 + 31 && k0 + 31 > warp_krow0 - p.window;
        uint32_t v[32];
        if (live) {
          tmem_ld_32x32(s_addr + sb * BLOCK_N, v);
          tmem_ld_wait();
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(bar_s_empty + 16 * map + 8 * sb);
        float bm = -INFINITY;
        if (live) {
          // scores in log2 units
          if (capped) {
            float top = 0.f;
#pragma unroll
            for (int i = 0; i < 32; i += 2) top = fmax3(top, fabsf(__uint_as_float(v[i])), fabsf(__uint_as_float(v[i + 1])));
            if (!__any_sync(0xffffffffu, top >= small_s)) {
#pragma unroll
              for (int i = 0; i < 32; i += 2) {
                const float2 c = cap_small(make_float2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), p.to_z, p.cap_log2e);
                v[i] = __float_as_uint(c.x), v[i + 1] = __float_as_uint(c.y);
              }
            } else {
#pragma unroll
              for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(cap_any(__uint_as_float(v[i]), p.to_z, p.cap_log2e));
            }
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * p.scale_log2e);
          }
          if (k0 + 31 > warp_krow0 || k0 <= warp_krow0 + 31 - p.window) {
            const int lim = krow - k0, low = lim - p.window;  // keys low < i <= lim are visible to this row
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              if (i > lim || i <= low) v[i] = 0xff800000u;
              bm = fmaxf(bm, __uint_as_float(v[i]));
            }
          } else {
            float b1 = -INFINITY;
#pragma unroll
            for (int i = 0; i < 32; i += 4) {
              bm = fmax3(bm, __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
              b1 = fmax3(b1, __uint_as_float(v[i + 2]), __uint_as_float(v[i + 3]));
            }
            bm = fmaxf(bm, b1);
          }
        }
        // the row's block maximum is the larger of its two halves (alternating slots: a thread is at most one exchange ahead)
        my_x[(it_count & 1) * 2 * BLOCK_M] = bm;
        __syncwarp();
        if (lane == 0) mbar_arrive(my_pair_bar);
        if (!mbar_wait(my_pair_bar, xphase, abort_flag, p.status_word, 68)) {
          alive = false;
          break;
        }
        xphase ^= 1u;
        bm = fmaxf(bm, partner_x[(it_count & 1) * 2 * BLOCK_M]);
        float m_new = fmaxf(m_run, bm);
        const float m_old = m_run;
        m_run = m_new;
        if (m_new == -INFINITY) m_new = 0.f;  // nothing in this row's window yet
        const float mult = ex2f(m_old - m_new);
        // the block before's P V read the P tile and produced the O that are about to change
        if (j > 0 && !mbar_wait(bar_pv_done + 8 * map, (it_count - 1) & 1, abort_flag, p.status_word, 69)) {
          alive = false;
          break;
        }
        tc_fence_after();
        float psum0 = 0.f, psum1 = 0.f;
        if (live) {
          uint32_t pk[16];
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const float p0 = ex2f(__uint_as_float(v[i]) - m_new), p1 = ex2f(__uint_as_float(v[i + 1]) - m_new);
            psum0 += p0;
            psum1 += p1;
            __half2 h = __floats2half2_rn(p0, p1);
            pk[i / 2] = *reinterpret_cast<uint32_t*>(&h);
          }
#pragma unroll
          for (int g = 0; g < 4; ++g)
            st_shared_v4(p_row + ((((uint32_t)(half * 4 + g)) ^ sw) << 4), pk[4 * g], pk[4 * g + 1], pk[4 * g + 2], pk[4 * g + 3]);
        } else if (warp_live) {
#pragma unroll
          for (int g = 0; g < 4; ++g) st_shared_v4(p_row + ((((uint32_t)(half * 4 + g)) ^ sw) << 4), 0u, 0u, 0u, 0u);
        }
        if (j > 0 && warp_live && __any_sync(0xffffffffu, mult != 1.0f)) {
#pragma unroll 1
          for (int c = 0; c < VD / 64; ++c) {
            uint32_t a[32];
            tmem_ld_32x32(o_addr + c * 32, a);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) a[i] = __float_as_uint(__uint_as_float(a[i]) * mult);
            tmem_st_32x32(o_addr + c * 32, a);
          }
          tmem_st_wait();
        }
        tc_fence_before();
        fence_proxy_async_smem();
        __syncwarp();
        if (lane == 0) mbar_arrive(bar_p_full + 8 * map);
        l_run = l_run * mult + (psum0 + psum1);
      }
      if (!alive) break;
      // both maps' last products, then the difference
      row_l[(map * 2 + half) * BLOCK_M + r_in_tile] = l_run;
      if (!meet()) break;
      if (!mbar_wait(bar_pv_done, (it_count - 1) & 1, abort_flag, p.status_word, 70)) break;
      if (!mbar_wait(bar_pv_done + 8, (it_count - 1) & 1, abort_flag, p.status_word, 71)) break;
      tc_fence_after();
      const float r0 = 1.0f / (row_l[r_in_tile] + row_l[BLOCK_M + r_in_tile]);
      const float r1 = -lambda / (row_l[2 * BLOCK_M + r_in_tile] + row_l[3 * BLOCK_M + r_in_tile]);
      constexpr int CQ = VD / 4;  // this thread's columns of the row
      const int c0 = (map * 2 + half) * CQ;
      float o[CQ], sq = 0.f;
      if (warp_live) {
#pragma unroll
        for (int c = 0; c < CQ; c += 16) {
          uint32_t a[16];
          tmem_ld_32x16(tmem_o + lane_addr + (uint32_t)(c0 + c), a);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[c + i] = __uint_as_float(a[i]) * r0;
          tmem_ld_32x16(tmem_o + lane_addr + (uint32_t)(VD + c0 + c), a);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[c + i] = fmaf(__uint_as_float(a[i]), r1, o[c + i]);
        }
#pragma unroll
        for (int i = 0; i < CQ; ++i) sq = fmaf(o[i], o[i], sq);  // (columns beyond vdim are zero)
      }
      row_sq[(map * 2 + half) * BLOCK_M + r_in_tile] = sq;
      // everyone who passes has the accumulators of these rows in registers: the next item's products may overwrite them
      tc_fence_before();
      if (!meet()) break;
      tc_fence_after();
      if (warp_live && row < w.q_end) {
        sq = (row_sq[r_in_tile] + row_sq[BLOCK_M + r_in_tile]) + (row_sq[2 * BLOCK_M + r_in_tile] + row_sq[3 * BLOCK_M + r_in_tile]);
        const int64_t grow = (int64_t)w.b * p.L + row;
        const float f = p.out_scale / sqrtf(sq / (float)p.vdim + p.eps) * __bfloat162float(p.gate[grow * p.ld_gate + w.h]);
        __nv_bfloat16* dst = p.out + grow * p.ld_out + (int64_t)w.h * p.vdim + c0;
        const int room = p.vdim - c0;  // (a multiple of 8)
#pragma unroll
        for (int g = 0; g < CQ / 8; ++g) {
          if (g * 8 < room) {
            uint32_t pk[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) pk[i] = pack_out<__nv_bfloat16>(o[g * 8 + 2 * i] * f, o[g * 8 + 2 * i + 1] * f);
            *reinterpret_cast<uint4*>(dst + g * 8) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
          }
        }
      }
    }
  }

  // ------------------------------------------------------------ teardown
  __syncwarp();
  if (*abort_flag) {
    const long long t0 = clock64();
    while (clock64() - t0 < 2000000LL) {
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM);
  }
}

template <int KD, int VD>
static int launch_sized(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const Args& a, cudaStream_t stream) {
  auto* kernel = pair_attention_sm100_kernel<KD, VD>;
  constexpr int smem = Shape<KD, VD>::SMEM;
  static std::atomic<bool> attr_set[kMaxDevices];
  const int slot = device_slot();
  if (slot < 0) return B200_ERR_CUDA;
  if (!attr_set[slot].load(std::memory_order_acquire)) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return B200_ERR_CUDA;
    attr_set[slot].store(true, std::memory_order_release);
  }
  const int64_t items = (int64_t)((a.L + BLOCK_M - 1) / BLOCK_M) * a.B * a.H;
  const int64_t grid = items < sm_count() ? items : sm_count();
  LaunchSetup ls(dim3((unsigned)grid), dim3(THREADS), smem, stream);
  const cudaError_t e = cudaLaunchKernelEx(&ls.cfg, kernel, mq, mk, mv, a, idesc(1, 1, 0, BLOCK_N), idesc(0, 0, 1, VD));
  note_launches(1);
  return status_from_cuda(e);
}

}  // namespace pair100

bool pair_attention_sm100_takes(int64_t dim, int64_t vdim, int dtype) {
  return dtype == B200_BF16 && dim <= 128 && vdim <= 128 && dim % 8 == 0 && vdim % 8 == 0;
}

int launch_pair_attention_sm100(const b200_pair_attention_args& p, cudaStream_t stream) {
  using namespace pair100;
  if (!pair_attention_sm100_takes(p.dim, p.vdim, p.dtype) || p.v_dtype != B200_F16 || p.pos_dev || !(p.scale > 0.f)) return B200_ERR_UNSUPPORTED;
  const int64_t keys = p.hist + p.n;
  const int64_t qs[3] = {p.n * p.ld_q, p.dim, p.ld_q}, ks[3] = {p.k_batch, p.dim, p.k_row}, vs[3] = {p.v_batch, p.v_head, p.v_row};
  if (p.k_head != 2 * p.dim || !view_ok(p.q, qs, p.B, 0) || !view_ok(p.k, ks, p.B, 0) || !view_ok(p.v, vs, p.B, 0) || (reinterpret_cast<uintptr_t>(p.out) & 15) || p.ld_out % 8)
    return B200_ERR_UNSUPPORTED;
  if (2 * p.B * p.heads > 0x7fffffffLL || keys > 0x7fffff00LL) return B200_ERR_UNSUPPORTED;
  CUtensorMap mq, mk, mv;
  Args a;
  int st = make_map(&mq, p.q, p.B, 2 * p.heads, p.n, p.dim, qs, BLOCK_M, B200_BF16, &a.q_head_inner);
  if (st == B200_OK) st = make_map(&mk, p.k, p.B, 2 * p.kv_heads, keys, p.dim, ks, BLOCK_N, B200_BF16, &a.k_head_inner);
  if (st == B200_OK) st = make_map(&mv, p.v, p.B, p.kv_heads, keys, p.vdim, vs, BLOCK_N, B200_F16, &a.v_head_inner);
  if (st != B200_OK) return B200_ERR_UNSUPPORTED;
  a.out = static_cast<__nv_bfloat16*>(p.out), a.ld_out = p.ld_out;
  a.gate = static_cast<const __nv_bfloat16*>(p.gate), a.ld_gate = p.ld_gate;
  a.lambda = p.lambda;
  a.B = (int)p.B, a.H = (int)p.heads, a.group = (int)(p.heads / p.kv_heads), a.L = (int)p.n, a.hist = (int)p.hist;
  a.window = (int)(p.window < keys ? p.window : keys), a.vdim = (int)p.vdim;
  const float log2e = 1.4426950408889634f;
  a.scale_log2e = p.scale * log2e;
  a.to_z = p.softcap > 0.f ? p.scale / p.softcap : 0.f, a.cap_log2e = p.softcap > 0.f ? p.softcap * log2e : 0.f;
  a.eps = p.eps, a.out_scale = p.out_scale;
  a.status_word = p.status_word;
  if (p.dim <= 64 && p.vdim <= 64) return launch_sized<64, 64>(mq, mk, mv, a, stream);
  if (p.dim <= 64) return launch_sized<64, 128>(mq, mk, mv, a, stream);
  return launch_sized<128, 128>(mq, mk, mv, a, stream);
}

}  // namespace b200
