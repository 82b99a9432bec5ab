// Building blocks of the tensor-core kernels that work on 128-row tiles in the panelled, 128-byte-swizzled layout
// (attention_tc.cu, layers_attn_tc.cu, layers_ssd.cu): bounded waits, tile loads, operand stores, the MMA loops.
#pragma once
#include <type_traits>

#include "sm100_common.cuh"

namespace gb {

template <typename T> struct OperandFmt { static constexpr int value = std::is_same<T, __nv_bfloat16>::value ? 1 : 0; };

constexpr int AT_M = 128;        // query rows per tile
constexpr int AT_N = 128;        // keys per tile

__device__ __forceinline__ bool at_wait(uint64_t* bar, uint32_t parity, int* status, int code, volatile int* abort_flag) {
  const long long t0 = clock64();
  for (;;) {
#pragma unroll 1
    for (int i = 0; i < 1024; ++i)
      if (mbar_try_wait(bar, parity)) return true;
    if (*abort_flag) return false;
    if (clock64() - t0 > 4000000000LL) {
      atomicCAS(status, 0, code);
      *abort_flag = 1;
      return false;
    }
  }
}

// [rows x 64] 16-bit tile with 128-byte rows, 128B swizzle: byte offset of element (r, c), c < 64
__device__ __forceinline__ uint32_t sw128_off(int r, int c) {
  return (uint32_t)(r * 128 + ((((c >> 3) ^ (r & 7)) << 4) | ((c & 7) << 1)));
}

// write 32 consecutive columns [c0, c0+32) of row r into a [128 x 128] operand buffer made of two 64-column panels
template <typename T>
__device__ __forceinline__ void store_p_chunk(uint8_t* sP, int r, int c0, const float (&v)[32]) {
  uint8_t* panel = sP + (c0 >> 6) * (AT_M * 128);
  const int cc = c0 & 63;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    uint4 q;
    q.x = Cvt<T>::pack2(v[8 * j + 0], v[8 * j + 1]);
    q.y = Cvt<T>::pack2(v[8 * j + 2], v[8 * j + 3]);
    q.z = Cvt<T>::pack2(v[8 * j + 4], v[8 * j + 5]);
    q.w = Cvt<T>::pack2(v[8 * j + 6], v[8 * j + 7]);
    *reinterpret_cast<uint4*>(panel + sw128_off(r, cc + 8 * j)) = q;
  }
}

// TMA load of a [128 rows x HD] tile as HD/64 panels
template <int HD>
__device__ __forceinline__ void load_tile(const CUtensorMap* tm, uint64_t* bar, uint8_t* dst, int col0, int row0) {
#pragma unroll
  for (int p = 0; p < HD / 64; ++p) tma_load_2d(tm, bar, dst + p * (AT_M * 128), col0 + 64 * p, row0);
}

// D[128 x N] (+)= A[128 x K] * B, all operands in the panelled SW128 layout.
//   a_kmajor tile: K runs along the 64-column panels.   b_mn: B given as [K rows x N cols] (N contiguous).
template <int KDIM>
__device__ __forceinline__ void mma_kmajor_kmajor(uint32_t tmem_d, uint32_t sa, uint32_t sb, uint32_t idesc, bool accumulate) {
  // A: [128 x KDIM] K-major, B: [N x KDIM] K-major
#pragma unroll
  for (int kk = 0; kk < KDIM / 16; ++kk) {
    const uint32_t off = (kk >> 2) * (AT_M * 128) + (kk & 3) * 32;
    umma_f16(tmem_d, make_smem_desc_sw128(sa + off, 16, 1024), make_smem_desc_sw128(sb + off, 16, 1024), idesc,
             (accumulate || kk > 0) ? 1u : 0u);
  }
}
template <int KDIM>
__device__ __forceinline__ void mma_kmajor_mnmajor(uint32_t tmem_d, uint32_t sa, uint32_t sb, uint32_t idesc, bool accumulate) {
  // A: [128 x KDIM] K-major (panels of 64 along K), B: [KDIM rows x N] with N contiguous (panels of 64 along N)
#pragma unroll
  for (int kk = 0; kk < KDIM / 16; ++kk) {
    const uint32_t aoff = (kk >> 2) * (AT_M * 128) + (kk & 3) * 32;
    const uint32_t boff = kk * 2048;   // 16 rows of 128 bytes
    umma_f16(tmem_d, make_smem_desc_sw128(sa + aoff, 16, 1024), make_smem_desc_sw128(sb + boff, AT_N * 128, 1024), idesc,
             (accumulate || kk > 0) ? 1u : 0u);
  }
}

}  // namespace gb
