// Differential attention of one token per sequence on tensor cores (bf16): the query heads of a key/value head share its
// cached keys and values, so a block takes up to 8 of them, both maps, and streams a range of the window once.
//
// One 16-row MMA tile holds map 0 of the heads in rows 0-7 and map 1 in rows 8-15: the scores of the two maps come from two
// products whose A operands are zero in the other's rows, and one P V serves both.  Keys and values go from global memory to
// MMA fragments without shared memory: a dot product does not care about the order of its columns, so a lane's 16 bytes of a
// key row are its elements of two k-steps (the queries are taken in the same order), and a lane's 16 bytes of four value rows
// are its elements of eight 8-column tiles (the output columns are put back in order when they are stored).  The softmax
// weights are fp32 by definition and enter their MMA as two bf16 parts.
//
// The blocks that share a (sequence, key/value head) form a cluster; its partial results meet in distributed shared memory.
#include "mma_sync.cuh"
#include "sm100_primitives.cuh"

namespace b200 {
namespace {

using namespace warp_mma;

constexpr int kWarps = 4, kHeads = 8, kKeys = 16;

__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float ld_cluster(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ uint32_t word_of(const uint4& v, int i) { return i == 0 ? v.x : i == 1 ? v.y : i == 2 ? v.z : v.w; }

// DG: 32-column groups of a query/key map, VG: 64-column groups of a value row.
template <int DG, int VG>
__global__ void __launch_bounds__(32 * kWarps, DG + VG <= 4 ? 3 : 2)
pair_decode_kernel(b200_pair_attention_args p, int head_tiles, int splits, float scale_log2e, float cap_log2e) {
  constexpr int VD = VG * 64, PITCH = VD + 4;
  __shared__ float part_o[kWarps][16][PITCH];
  __shared__ float part_m[kWarps][16], part_l[kWarps][16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3;
  const int rank = blockIdx.x;  // cluster = the blocks of one grid row
  const int ht = blockIdx.y % head_tiles;
  const int64_t g = (blockIdx.y / head_tiles) % p.kv_heads, b = blockIdx.y / (head_tiles * p.kv_heads);
  const int group = (int)(p.heads / p.kv_heads), nh = min(kHeads, group - ht * kHeads);
  const int64_t h0 = g * group + ht * kHeads;
  const int dim = (int)p.dim, vdim = (int)p.vdim, ring = (int)p.ring;
  const int64_t pos = p.pos_dev[0];
  const int n_keys = (int)(pos + 1 < p.window ? pos + 1 : p.window);
  const int first = (int)((pos + 1 - n_keys) % ring);
  const auto* kb = static_cast<const __nv_bfloat16*>(p.k) + b * p.k_batch + g * p.k_head;
  const auto* vb = static_cast<const __nv_bfloat16*>(p.v) + b * p.v_batch + g * p.v_head;
  const uint4 zero = make_uint4(0, 0, 0, 0);

  auto slot_of = [&](int j) {
    const int s = first + j;
    return s >= ring ? s - ring : s;
  };
  uint4 k[2][2][DG], v[VG][4];
  auto load_k = [&](int tile) {
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int j = tile * kKeys + nt * 8 + g8;
      const auto* row = kb + (int64_t)slot_of(j) * p.k_row;
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int i = 0; i < DG; ++i) {
          const int c = i * 32 + t4 * 8;
          k[nt][m][i] = j < n_keys && c < dim ? __ldg(reinterpret_cast<const uint4*>(row + m * dim + c)) : zero;
        }
    }
  };
  auto load_v = [&](int tile) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int j = tile * kKeys + t4 * 2 + (e & 1) + (e >> 1) * 8;
      const auto* row = vb + (int64_t)slot_of(j) * p.v_row;
#pragma unroll
      for (int i = 0; i < VG; ++i) {
        const int c = i * 64 + g8 * 8;
        v[i][e] = j < n_keys && c < vdim ? __ldg(reinterpret_cast<const uint4*>(row + c)) : zero;
      }
    }
  };
  const int tiles = (n_keys + kKeys - 1) / kKeys, step = splits * kWarps;
  int tile = rank * kWarps + warp;
  if (tile < tiles) load_k(tile), load_v(tile);

  uint4 q[2][DG];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int i = 0; i < DG; ++i) {
      const int c = i * 32 + t4 * 8;
      const auto* src = static_cast<const __nv_bfloat16*>(p.q) + b * p.ld_q + ((h0 + g8) * 2 + m) * dim + c;
      q[m][i] = g8 < nh && c < dim ? *reinterpret_cast<const uint4*>(src) : zero;
    }

  float o[VG * 8][4];
#pragma unroll
  for (int i = 0; i < VG * 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  const float to_2z = p.softcap > 0.f ? p.scale / p.softcap * 2.8853900817779268f : 0.f;
  for (; tile < tiles; tile += step) {
    float s[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
#pragma unroll
      for (int i = 0; i < DG; ++i) {
        const uint32_t a0[4] = {q[0][i].x, 0, q[0][i].y, 0}, a1[4] = {q[0][i].z, 0, q[0][i].w, 0};
        const uint32_t a2[4] = {0, q[1][i].x, 0, q[1][i].y}, a3[4] = {0, q[1][i].z, 0, q[1][i].w};
        mma_bf16(s[nt], a0, k[nt][0][i].x, k[nt][0][i].y);
        mma_bf16(s[nt], a1, k[nt][0][i].z, k[nt][0][i].w);
        mma_bf16(s[nt], a2, k[nt][1][i].x, k[nt][1][i].y);
        mma_bf16(s[nt], a3, k[nt][1][i].z, k[nt][1][i].w);
      }
    }
    const int j0 = tile * kKeys;
    if (tile + step < tiles) load_k(tile + step);
    // scores in log2 units; keys beyond the last: no weight
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float x = s[nt][e];
        if (cap_log2e > 0.f) {
          float r;
          asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + ex2_fast(x * to_2z)));
          x = fmaf(-2.0f * cap_log2e, r, cap_log2e);
        } else {
          x *= scale_log2e;
        }
        x = j0 + nt * 8 + t4 * 2 + (e & 1) < n_keys ? x : -INFINITY;
        s[nt][e] = x;
        mx[e >> 1] = fmaxf(mx[e >> 1], x);
      }
    float mult[2];
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      mx[m] = fmaxf(mx[m], __shfl_xor_sync(0xffffffffu, mx[m], 1));
      mx[m] = fmaxf(mx[m], __shfl_xor_sync(0xffffffffu, mx[m], 2));
      const float m_new = fmaxf(m_run[m], mx[m]);  // (the first key of a tile always exists: finite)
      mult[m] = ex2_fast(m_run[m] - m_new);
      m_run[m] = m_new;
    }
    uint32_t ph[4], pl[4];
    float sum[2] = {0.f, 0.f};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const float p0 = ex2_fast(s[nt][2 * m] - m_run[m]), p1 = ex2_fast(s[nt][2 * m + 1] - m_run[m]);
        sum[m] += p0 + p1;
        split_pair(p0, p1, ph[nt * 2 + m], pl[nt * 2 + m]);
      }
    l_run[0] = fmaf(l_run[0], mult[0], sum[0]), l_run[1] = fmaf(l_run[1], mult[1], sum[1]);
    if (__any_sync(0xffffffffu, mult[0] != 1.0f || mult[1] != 1.0f)) {
#pragma unroll
      for (int i = 0; i < VG * 8; ++i) o[i][0] *= mult[0], o[i][1] *= mult[0], o[i][2] *= mult[1], o[i][3] *= mult[1];
    }
#pragma unroll
    for (int i = 0; i < VG; ++i)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const uint32_t sel = (j & 1) ? 0x7632u : 0x5410u;
        const uint32_t b0 = __byte_perm(word_of(v[i][0], j >> 1), word_of(v[i][1], j >> 1), sel);
        const uint32_t b1 = __byte_perm(word_of(v[i][2], j >> 1), word_of(v[i][3], j >> 1), sel);
        mma_bf16(o[i * 8 + j], ph, b0, b1);
        mma_bf16(o[i * 8 + j], pl, b0, b1);
      }
    if (tile + step < tiles) load_v(tile + step);
  }
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    l_run[m] += __shfl_xor_sync(0xffffffffu, l_run[m], 1);
    l_run[m] += __shfl_xor_sync(0xffffffffu, l_run[m], 2);
    if (t4 == 0) part_m[warp][m * 8 + g8] = m_run[m], part_l[warp][m * 8 + g8] = l_run[m];
  }
#pragma unroll
  for (int i = 0; i < VG; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) part_o[warp][g8 + (e >> 1) * 8][i * 64 + (t4 * 2 + (e & 1)) * 8 + j] = o[i * 8 + j][e];
  __syncthreads();
  // the block's warps into the first one's place: four rows per warp
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = warp * 4 + i;
    float m = part_m[0][r], f[kWarps], l = 0.f;
#pragma unroll
    for (int w = 1; w < kWarps; ++w) m = fmaxf(m, part_m[w][r]);
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      f[w] = m == -INFINITY ? 0.f : ex2_fast(part_m[w][r] - m);
      l = fmaf(part_l[w][r], f[w], l);
    }
    for (int c = lane; c < VD; c += 32) {
      float a = 0.f;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) a = fmaf(part_o[w][r][c], f[w], a);
      part_o[0][r][c] = a;
    }
    __syncwarp();
    if (lane == 0) part_m[0][r] = m, part_l[0][r] = l;
  }
  if (splits > 1) sm100::cluster_sync_all();
  else __syncthreads();
  // head i of the tile: block i % splits, warp (i / splits) % 4; the cluster's partial results, the difference, norm and gate
  const float lambda = __ldg(p.lambda);
  for (int i = rank + splits * warp; i < nh; i += splits * kWarps) {
    float total[VD / 32];
#pragma unroll
    for (int c = 0; c < VD / 32; ++c) total[c] = 0.f;
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const int r = m * 8 + i;
      const uint32_t am = (uint32_t)__cvta_generic_to_shared(&part_m[0][r]), al = (uint32_t)__cvta_generic_to_shared(&part_l[0][r]);
      const uint32_t ao = (uint32_t)__cvta_generic_to_shared(&part_o[0][r][lane]);
      float top = -INFINITY;
      for (int s = 0; s < splits; ++s) top = fmaxf(top, ld_cluster(sm100::mapa_shared(am, s)));
      float l = 0.f, a[VD / 32];
#pragma unroll
      for (int c = 0; c < VD / 32; ++c) a[c] = 0.f;
      for (int s = 0; s < splits; ++s) {
        const float f = ex2_fast(ld_cluster(sm100::mapa_shared(am, s)) - top);
        l = fmaf(ld_cluster(sm100::mapa_shared(al, s)), f, l);
        const uint32_t row = sm100::mapa_shared(ao, s);
#pragma unroll
        for (int c = 0; c < VD / 32; ++c) a[c] = fmaf(ld_cluster(row + c * 128), f, a[c]);
      }
      const float w = (m ? -lambda : 1.0f) / l;
#pragma unroll
      for (int c = 0; c < VD / 32; ++c) total[c] = fmaf(a[c], w, total[c]);
    }
    float sq = 0.f;
#pragma unroll
    for (int c = 0; c < VD / 32; ++c) sq = fmaf(total[c], total[c], sq);  // (columns beyond vdim are zero)
    const int64_t h = h0 + i;
    const float f = p.out_scale / sqrtf(warp_sum(sq) / (float)vdim + p.eps) * __bfloat162float(static_cast<const __nv_bfloat16*>(p.gate)[b * p.ld_gate + h]);
    auto* out = static_cast<__nv_bfloat16*>(p.out) + b * p.ld_out + h * vdim;
#pragma unroll
    for (int c = 0; c < VD / 32; ++c)
      if (c * 32 + lane < vdim) out[c * 32 + lane] = __float2bfloat16_rn(total[c] * f);
  }
  if (splits > 1) sm100::cluster_sync_all();  // nobody leaves while its partial results are being read
}

// Blocks per (sequence, key/value head, head tile): the fewest rounds of blocks, counted in tiles of 16 keys per warp.
int split_count(int64_t rows, int64_t window, int per_sm) {
  const int64_t tiles = (window + kKeys - 1) / kKeys, slots = (int64_t)sm_count() * per_sm;
  int best = 1;
  double cost = 0;
  for (int s = 1; s <= 8; s *= 2) {
    const double c = (double)((rows * s + slots - 1) / slots) * ((double)((tiles + s * kWarps - 1) / (s * kWarps)) + 2.0);
    if (s == 1 || c < cost) cost = c, best = s;
  }
  return best;
}

template <int DG, int VG>
int launch_sized(const b200_pair_attention_args& p, cudaStream_t stream) {
  const int64_t group = p.heads / p.kv_heads, head_tiles = (group + kHeads - 1) / kHeads, rows = p.B * p.kv_heads * head_tiles;
  if (rows > 65535) return B200_ERR_UNSUPPORTED;
  const int splits = split_count(rows, p.window, DG + VG <= 4 ? 3 : 2);
  const float log2e = 1.4426950408889634f;
  LaunchSetup ls(dim3((unsigned)splits, (unsigned)rows), dim3(32 * kWarps), 0, stream, splits, false);
  const cudaError_t e = cudaLaunchKernelEx(&ls.cfg, pair_decode_kernel<DG, VG>, p, (int)head_tiles, splits, p.scale * log2e,
                                           p.softcap > 0.f ? p.softcap * log2e : 0.f);
  note_launches(1);
  return status_from_cuda(e);
}

}  // namespace

int launch_pair_decode(const b200_pair_attention_args& p, cudaStream_t stream) {
  if (!p.pos_dev || p.dtype != B200_BF16 || p.v_dtype != B200_BF16 || p.dim > 128 || p.vdim > 128 || p.dim % 8 || p.vdim % 8) return B200_ERR_UNSUPPORTED;
  if (((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.k) | reinterpret_cast<uintptr_t>(p.v)) & 15) || p.ld_q % 8 || p.k_row % 8 || p.v_row % 8 ||
      p.k_batch % 8 || p.k_head % 8 || p.v_batch % 8 || p.v_head % 8)
    return B200_ERR_UNSUPPORTED;
  const int dg = (int)(p.dim + 31) / 32, vg = (int)(p.vdim + 63) / 64;
  switch (dg * 2 + vg) {
    case 3: return launch_sized<1, 1>(p, stream);
    case 4: return launch_sized<1, 2>(p, stream);
    case 5: return launch_sized<2, 1>(p, stream);
    case 6: return launch_sized<2, 2>(p, stream);
    case 7: return launch_sized<3, 1>(p, stream);
    case 8: return launch_sized<3, 2>(p, stream);
    case 9: return launch_sized<4, 1>(p, stream);
    default: return launch_sized<4, 2>(p, stream);
  }
}

}  // namespace b200
