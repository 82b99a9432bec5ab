// Small helpers shared by the kernels of layer-list models.
#pragma once
#include "sm100_common.cuh"
#include "gb_layers.h"

namespace gb {

__device__ __forceinline__ float ll_inv_rms(float sum_sq, int n, float eps) { return 1.0f / sqrtf(sum_sq / (float)n + eps); }
__device__ __forceinline__ float ll_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float ll_silu(float z) { return z / (1.0f + expf(-z)); }
// The same for results that are rounded to 16 bits: hardware exponential and reciprocal (relative error about 2^-21).
__device__ __forceinline__ float ll_sigmoid_fast(float z) { return __fdividef(1.0f, 1.0f + __expf(fminf(-z, 80.f))); }
template <typename T> __device__ __forceinline__ float ll_sigmoid_t(float z) {
  if constexpr (sizeof(T) == 4) return ll_sigmoid(z);
  else return ll_sigmoid_fast(z);
}
template <typename T> __device__ __forceinline__ float ll_silu_t(float z) {
  if constexpr (sizeof(T) == 4) return ll_silu(z);
  else return z * ll_sigmoid_fast(z);
}
// eight consecutive values
__device__ __forceinline__ void ll_load8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 q = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) { const float2 f = Cvt<__nv_bfloat16>::unpack2(w[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
}
__device__ __forceinline__ void ll_load8(const float* p, float (&v)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void ll_store8(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 q;
  q.x = Cvt<__nv_bfloat16>::pack2(v[0], v[1]); q.y = Cvt<__nv_bfloat16>::pack2(v[2], v[3]);
  q.z = Cvt<__nv_bfloat16>::pack2(v[4], v[5]); q.w = Cvt<__nv_bfloat16>::pack2(v[6], v[7]);
  *reinterpret_cast<uint4*>(p) = q;
}
__device__ __forceinline__ void ll_store8(float* p, const float (&v)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
// eight consecutive values as stored
template <typename T> struct LlRaw8;
template <> struct LlRaw8<__nv_bfloat16> {
  uint4 q;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { q = __ldg(reinterpret_cast<const uint4*>(p)); }
  __device__ __forceinline__ void expand(float (&v)[8]) const {
    const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = Cvt<__nv_bfloat16>::unpack2(w[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
  }
};
template <> struct LlRaw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) {
    a = __ldg(reinterpret_cast<const float4*>(p));
    b = __ldg(reinterpret_cast<const float4*>(p) + 1);
  }
  __device__ __forceinline__ void expand(float (&v)[8]) const {
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
};
// log(1 + e^z), without overflow for large z
__device__ __forceinline__ float ll_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// four consecutive values, raw and expanded
template <typename T> struct LlRaw4;
template <> struct LlRaw4<__nv_bfloat16> {
  uint2 q;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { q = *reinterpret_cast<const uint2*>(p); }
  __device__ __forceinline__ void expand(float (&v)[4]) const {
    const float2 a = Cvt<__nv_bfloat16>::unpack2(q.x), b = Cvt<__nv_bfloat16>::unpack2(q.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const { *reinterpret_cast<uint2*>(p) = q; }
};
template <> struct LlRaw4<float> {
  float4 q;
  __device__ __forceinline__ void load(const float* p) { q = *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ void expand(float (&v)[4]) const { v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = q; }
};
__device__ __forceinline__ void ll_store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void ll_store4(__nv_bfloat16* p, const float4& v) {
  uint2 q;
  q.x = Cvt<__nv_bfloat16>::pack2(v.x, v.y);
  q.y = Cvt<__nv_bfloat16>::pack2(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = q;
}

// V neighbouring values
__device__ __forceinline__ void ll_get(const float* p, float (&v)[4]) {
  const float4 q = *reinterpret_cast<const float4*>(p);
  v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
}
__device__ __forceinline__ void ll_get(const __nv_bfloat16* p, float (&v)[4]) {
  LlRaw4<__nv_bfloat16> r;
  r.load(p);
  r.expand(v);
}
template <typename T> __device__ __forceinline__ void ll_get(const T* p, float (&v)[8]) { ll_load8(p, v); }
template <typename T> __device__ __forceinline__ void ll_get(const T* p, float (&v)[1]) { v[0] = Cvt<T>::to_f(*p); }
template <typename T> __device__ __forceinline__ void ll_put(T* p, const float (&v)[4]) { ll_store4(p, make_float4(v[0], v[1], v[2], v[3])); }
template <typename T> __device__ __forceinline__ void ll_put(T* p, const float (&v)[8]) { ll_store8(p, v); }
template <typename T> __device__ __forceinline__ void ll_put(T* p, const float (&v)[1]) { *p = Cvt<T>::from_f(v[0]); }

// sum over the TPR threads of a row (a warp, or the block of 256); every thread gets it
template <int TPR>
__device__ __forceinline__ float ll_row_sum(float v, float* red) {
  v = warp_sum(v);
  if constexpr (TPR > 32) {
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    v = 0.f;
#pragma unroll
    for (int i = 0; i < TPR / 32; ++i) v += red[i];
  }
  return v;
}

// Norm of one row by TPR threads, V neighbouring values at a time.  `get(i, v)` gives the values at i .. i + V - 1 and is
// called once per place, except for places past the ones kept in registers, which `again(i, v)` gives once more; `put(i, v)`
// takes the normed values.  KEEP * V values per thread stay in registers.
template <int TPR, int V, int KEEP, typename Get, typename Again, typename Put>
__device__ __forceinline__ void ll_row_norm(int d, int mode, const float* __restrict__ w, const float* __restrict__ b, float eps, float* red,
                                            Get get, Again again, Put put) {
  const int t = threadIdx.x % TPR;
  float keep[KEEP][V];
  float sum = 0.f, dev = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = (t + k * TPR) * V;
    if (i < d) get(i, keep[k]);
    else {
#pragma unroll
      for (int e = 0; e < V; ++e) keep[k][e] = 0.f;
    }
#pragma unroll
    for (int e = 0; e < V; ++e) sum += keep[k][e];
  }
  for (int i = (t + KEEP * TPR) * V; i < d; i += TPR * V) {
    float v[V];
    get(i, v);
#pragma unroll
    for (int e = 0; e < V; ++e) sum += v[e];
  }
  const float mean = mode == GB_LL_NORM_LAYER ? ll_row_sum<TPR>(sum, red) / (float)d : 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k)
    if ((t + k * TPR) * V < d) {
#pragma unroll
      for (int e = 0; e < V; ++e) { const float c = keep[k][e] - mean; dev += c * c; }
    }
  for (int i = (t + KEEP * TPR) * V; i < d; i += TPR * V) {
    float v[V];
    again(i, v);
#pragma unroll
    for (int e = 0; e < V; ++e) { const float c = v[e] - mean; dev += c * c; }
  }
  const float inv = ll_inv_rms(ll_row_sum<TPR>(dev, red), d, eps);
  auto finish = [&](int i, float (&v)[V]) {
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = (v[e] - mean) * inv;
    float u[V];
    ll_get(w + i, u);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] *= u[e];
    if (b) {
      ll_get(b + i, u);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += u[e];
    }
    put(i, v);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = (t + k * TPR) * V;
    if (i < d) finish(i, keep[k]);
  }
  for (int i = (t + KEEP * TPR) * V; i < d; i += TPR * V) {
    float v[V];
    again(i, v);
    finish(i, v);
  }
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
