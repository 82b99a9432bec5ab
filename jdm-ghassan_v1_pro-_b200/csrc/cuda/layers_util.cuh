// Small helpers shared by the kernels of layer-list models.
#pragma once
#include "sm100_common.cuh"

namespace gb {

__device__ __forceinline__ float ll_inv_rms(float sum_sq, int n, float eps) { return 1.0f / sqrtf(sum_sq / (float)n + eps); }
__device__ __forceinline__ float ll_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float ll_silu(float z) { return z / (1.0f + expf(-z)); }
// log(1 + e^z), without overflow for large z
__device__ __forceinline__ float ll_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ void ll_store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void ll_store4(__nv_bfloat16* p, const float4& v) {
  uint2 q;
  q.x = Cvt<__nv_bfloat16>::pack2(v.x, v.y);
  q.y = Cvt<__nv_bfloat16>::pack2(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = q;
}

// Cache row of a position: the first `keep` rows are never given up, the rest is a ring of cap - keep rows.
__device__ __forceinline__ int ll_ring_row(int p, int keep, int cap) { return p < keep ? p : keep + (p - keep) % (cap - keep); }

// kernel<<<grid, block, smem>>> with programmatic stream serialization, opting in to more than 48 KB of shared memory
#define GB_PDL_LAUNCH_SMEM(kernel, grid, block, smem, st, ...)                                                       \
  do {                                                                                                               \
    cudaLaunchAttribute gb_attr_;                                                                                    \
    cudaLaunchConfig_t gb_cfg_ = gb_pdl_config(grid, block, smem, st, &gb_attr_);                                    \
    if ((smem) > 48 * 1024) (void)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem)); \
    (void)cudaLaunchKernelEx(&gb_cfg_, kernel, __VA_ARGS__);                                                         \
  } while (0)

}  // namespace gb
