// What the tcgen05 attention kernels share: operand descriptors, query tiles, tensor-memory stores, tensor maps.
#pragma once

#include "sm100_primitives.cuh"

namespace b200 {
namespace attn100 {

using namespace sm100;

constexpr int BLOCK_M = 128;  // query rows per tile
constexpr int BLOCK_N = 64;   // keys per block

// K-major operand, 128-byte swizzle (rows of 128 bytes, 8-row groups of 1024 bytes).
__device__ __forceinline__ uint64_t desc_kmajor(uint32_t addr) {
  return (uint64_t)((addr & 0x3FFFF) >> 4) | ((uint64_t)1 << 16) | ((uint64_t)(1024 >> 4) << 32) | ((uint64_t)1 << 46) |
         ((uint64_t)2 << 61);
}
// MN-major operand, 128-byte swizzle: 64 contiguous MN elements per 128-byte row, 8 K-rows per 1024-byte
// group; groups along K are `stride byte offset` apart, 64-wide MN chunks `leading byte offset` (= one atom) apart.
// This is how a [keys, head_dim] V tile serves as the B operand of P V.
__device__ __forceinline__ uint64_t desc_mnmajor(uint32_t addr, int atom_bytes) {
  return (uint64_t)((addr & 0x3FFFF) >> 4) | ((uint64_t)(atom_bytes >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | ((uint64_t)1 << 46) |
         ((uint64_t)2 << 61);
}
// kind::f16 instruction descriptor: fp32 accumulator, M = 128, N = n.
__host__ __device__ constexpr uint32_t idesc(int a_fmt, int b_fmt, int b_mn_major, int n) {
  return (1u << 4) | ((uint32_t)a_fmt << 7) | ((uint32_t)b_fmt << 10) | ((uint32_t)b_mn_major << 16) | ((uint32_t)(n >> 3) << 17) |
         ((uint32_t)(BLOCK_M >> 4) << 24);
}

// Query rows [0, L) are cut into n_qt = ceil(L / 128) tiles of at most 128 rows whose ENDS are as early as they can be:
// tile i ends at min(L, round_up(L - 128 * (n_qt - 1 - i), 64)) and starts where tile i - 1 ends.  A tile costs one
// 64-key block per 64 rows up to its end, so a ragged L puts its short tile first, where the causal rows are
// shortest (L = 300: rows [0,64) [64,192) [192,300) = 1 + 3 + 5 key blocks, where [0,128) [128,256) [256,300) would
// take 2 + 4 + 5); starts stay multiples of 64, so only the last two key blocks of a tile need per-element masks.
// A tile always loads 128 rows of Q; rows at or beyond its end are computed and dropped.
// Items ordered by decreasing row-tile index (the longest causal rows first), then (batch, head).
__device__ __forceinline__ int tile_end(int i, int n_qt, int L) {
  const int e = (L - BLOCK_M * (n_qt - 1 - i) + BLOCK_N - 1) / BLOCK_N * BLOCK_N;
  return min(L, e);
}

__device__ __forceinline__ float fmax3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ float ex2f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void ld_shared_v4(uint32_t addr, uint32_t (&v)[4]) {
  asm volatile("ld.shared.v4.b32 {%0, %1, %2, %3}, [%4];" : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void st_shared_v4(uint32_t addr, uint32_t a, uint32_t b, uint32_t c, uint32_t d) {
  asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(addr), "r"(a), "r"(b), "r"(c), "r"(d) : "memory");
}
__device__ __forceinline__ void st_global_v8(void* p, const uint32_t* v) {
  asm volatile("st.global.v8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(p), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]),
               "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7])
               : "memory");
}
template <typename T>
__device__ __forceinline__ uint32_t pack_out(float a, float b);
template <>
__device__ __forceinline__ uint32_t pack_out<__half>(float a, float b) {
  __half2 h = __floats2half2_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}
template <>
__device__ __forceinline__ uint32_t pack_out<__nv_bfloat16>(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}

__device__ __forceinline__ void tmem_st_32x32(uint32_t taddr, const uint32_t (&v)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]),
        "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]), "r"(v[16]), "r"(v[17]), "r"(v[18]), "r"(v[19]), "r"(v[20]), "r"(v[21]),
        "r"(v[22]), "r"(v[23]), "r"(v[24]), "r"(v[25]), "r"(v[26]), "r"(v[27]), "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31])
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// 4-D map over a strided (batch, head, row) view with contiguous head_dim.  The two middle dimensions are
// ordered by ascending stride ({D, row, head, batch} for contiguous [B, NH, L, D] tensors, {D, head, row, batch}
// for views into a fused [B, L, 3*NH*D] projection); *head_inner tells the kernel which order was used.
inline int make_map(CUtensorMap* map, const void* ptr, int64_t B, int64_t NH, int64_t L, int64_t D, const int64_t* s, int box_rows, int dtype,
                    int* head_inner) {
  *head_inner = s[1] < s[2];
  uint64_t dims[4] = {(uint64_t)D, (uint64_t)L, (uint64_t)NH, (uint64_t)B};
  uint64_t strides[3] = {(uint64_t)s[2] * 2, (uint64_t)s[1] * 2, (uint64_t)s[0] * 2};
  uint32_t box[4] = {64, (uint32_t)box_rows, 1, 1};
  if (*head_inner) {
    dims[1] = (uint64_t)NH, dims[2] = (uint64_t)L;
    strides[0] = (uint64_t)s[1] * 2, strides[1] = (uint64_t)s[2] * 2;
    box[1] = 1, box[2] = (uint32_t)box_rows;
  }
  return encode_tensor_map(map, ptr, 4, dims, strides, box, dtype, CU_TENSOR_MAP_L2_PROMOTION_L2_256B);
}

inline bool view_ok(const void* ptr, const int64_t* s, int64_t B, int64_t NH) {
  if (reinterpret_cast<uintptr_t>(ptr) & 15) return false;
  // TMA wants 16-byte multiples for every stride; a stride of a size-1 dimension is never used but must still encode
  for (int i = 0; i < 3; ++i)
    if (s[i] % 8 != 0 || s[i] <= 0 || (uint64_t)s[i] * 2 >= (1ull << 40)) return false;
  (void)B;
  (void)NH;
  return true;
}

}  // namespace attn100
}  // namespace b200
