// Row-wise kernels of layer-list models (interface in gb_layers.h): embedding, norms on sublayer outputs with the residual
// add, residual adds with the norm ahead of the next sublayer, the fp32 matrix product, the fp32 SwiGLU and squared
// relu, the logit cap.
#include <type_traits>

#include "sm100_common.cuh"
#include "gb_layers.h"
#include "layers_util.cuh"

namespace gb {

template <typename T>
__global__ void ll_embed_kernel(const int* __restrict__ ids, const T* __restrict__ table, long long ld_table, int vocab,
                                float* __restrict__ x, T* __restrict__ x16, long long ld16, int rows, int d) {
  pdl_wait();
  const int r = blockIdx.x;
  const int id = ids[r];
  const bool ok = id >= 0 && id < vocab;
  for (int i = threadIdx.x; i < ld16; i += blockDim.x) {
    const T v = (ok && i < d) ? table[(long long)id * ld_table + i] : Cvt<T>::from_f(0.f);
    x16[(long long)r * ld16 + i] = v;
    if (i < d) x[(long long)r * d + i] = Cvt<T>::to_f(v);
  }
}

// One warp per row.  VEC: d a multiple of 4 and 16-byte aligned rows.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) ll_postnorm_kernel(const float* __restrict__ y, long long ldy, const float* x,
                                                          const float* __restrict__ w, float eps, float* x_out,
                                                          T* __restrict__ x16, long long ld16, int rows, int d) {
  pdl_wait();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  const float* yr = y + r * ldy;
  const float* xr = x + (long long)r * d;
  float* xo = x_out + (long long)r * d;
  float ss = 0.f;
  if constexpr (VEC) {
    constexpr int KEEP = 8;                       // float4 per lane kept in registers between the two passes
    const int n4 = d >> 2;
    float4 keep[KEEP], xk[KEEP];
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = lane + 32 * k;
      keep[k] = i < n4 ? reinterpret_cast<const float4*>(yr)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
      xk[k] = i < n4 ? reinterpret_cast<const float4*>(xr)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int k = 0; k < KEEP; ++k) ss += keep[k].x * keep[k].x + keep[k].y * keep[k].y + keep[k].z * keep[k].z + keep[k].w * keep[k].w;
    for (int i = lane + 32 * KEEP; i < n4; i += 32) {
      const float4 v = reinterpret_cast<const float4*>(yr)[i];
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float inv = ll_inv_rms(warp_sum(ss), d, eps);
    auto put = [&](int i, const float4& v, const float4& xv) {
      const float4 g = reinterpret_cast<const float4*>(w)[i];
      float4 o;
      o.x = xv.x + v.x * inv * g.x; o.y = xv.y + v.y * inv * g.y; o.z = xv.z + v.z * inv * g.z; o.w = xv.w + v.w * inv * g.w;
      reinterpret_cast<float4*>(xo)[i] = o;
      if (x16) ll_store4(x16 + (long long)r * ld16 + 4 * i, o);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = lane + 32 * k;
      if (i < n4) put(i, keep[k], xk[k]);
    }
    for (int i = lane + 32 * KEEP; i < n4; i += 32)
      put(i, reinterpret_cast<const float4*>(yr)[i], reinterpret_cast<const float4*>(xr)[i]);
  } else {
    for (int i = lane; i < d; i += 32) ss += yr[i] * yr[i];
    const float inv = ll_inv_rms(warp_sum(ss), d, eps);
    for (int i = lane; i < d; i += 32) {
      const float o = xr[i] + yr[i] * inv * w[i];
      xo[i] = o;
      if (x16) x16[(long long)r * ld16 + i] = Cvt<T>::from_f(o);
    }
  }
  if (x16)
    for (int i = d + lane; i < ld16; i += 32) x16[(long long)r * ld16 + i] = Cvt<T>::from_f(0.f);
}

template <typename T>
__global__ void __launch_bounds__(256) ll_norm_rows_kernel(const float* __restrict__ x, const int* __restrict__ row_idx,
                                                           const float* __restrict__ w, float eps, T* __restrict__ out,
                                                           long long ldo, int rows, int d) {
  pdl_wait();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  const float* xr = x + (long long)(row_idx ? row_idx[r] : r) * d;
  float ss = 0.f;
  for (int i = lane; i < d; i += 32) ss += xr[i] * xr[i];
  const float inv = ll_inv_rms(warp_sum(ss), d, eps);
  for (int i = lane; i < ldo; i += 32) out[r * ldo + i] = Cvt<T>::from_f(i < d ? xr[i] * inv * w[i] : 0.f);
}

template <typename T, int TPR, int V>
__global__ void __launch_bounds__(256) ll_embed_norm_kernel(const int* __restrict__ ids, const T* __restrict__ table, long long ld_table, int vocab,
                                                            int mode, const float* __restrict__ w, const float* __restrict__ b, float eps,
                                                            float* __restrict__ x, int rows, int d) {
  pdl_wait();
  __shared__ float red[8];
  const int r = TPR == 32 ? blockIdx.x * 8 + (threadIdx.x >> 5) : blockIdx.x;
  if (r >= rows) return;
  const int id = ids[r];
  const bool ok = id >= 0 && id < vocab;
  auto get = [&](int i, float (&v)[V]) {
    if (ok) ll_get(table + (long long)id * ld_table + i, v);
    else {
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = 0.f;
    }
  };
  ll_row_norm<TPR, V, 8>(d, mode, w, b, eps, red, get, get, [&](int i, const float (&v)[V]) { ll_put(x + (long long)r * d + i, v); });
}

template <typename T, int TPR, int V>
__global__ void __launch_bounds__(256) ll_add_norm_kernel(const float* __restrict__ y, long long ldy, float alpha, const float* x, const float* x0,
                                                          const int* __restrict__ row_idx, int mode, const float* __restrict__ w,
                                                          const float* __restrict__ b, float eps, float* x_out, T* __restrict__ out,
                                                          long long ldo, int rows, int d) {
  pdl_wait();
  __shared__ float red[8];
  const int r = TPR == 32 ? blockIdx.x * 8 + (threadIdx.x >> 5) : blockIdx.x;
  if (r >= rows) return;
  const long long src = (long long)(row_idx ? row_idx[r] : r) * d;
  auto add = [&](int i, float (&v)[V]) {
    ll_get(x + src + i, v);
    if (y) {
      float u[V];
      ll_get(y + (long long)r * ldy + i, u);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += alpha * u[e];
    }
    if (x0) {
      float u[V];
      ll_get(x0 + src + i, u);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += u[e];
    }
  };
  auto get = [&](int i, float (&v)[V]) {
    add(i, v);
    if (x_out) ll_put(x_out + (long long)r * d + i, v);
  };
  if (!out) {
    for (int i = (threadIdx.x % TPR) * V; i < d; i += TPR * V) {
      float v[V];
      get(i, v);
    }
    return;
  }
  ll_row_norm<TPR, V, 8>(d, mode, w, b, eps, red, get,
                      [&](int i, float (&v)[V]) { if (x_out) ll_get(x_out + (long long)r * d + i, v); else add(i, v); },
                      [&](int i, const float (&v)[V]) { ll_put(out + r * ldo + i, v); });
  for (int i = d + threadIdx.x % TPR; i < ldo; i += TPR) out[r * ldo + i] = Cvt<T>::from_f(0.f);
}

__global__ void ll_relu2_kernel(float* __restrict__ v, long long ld, int n) {
  pdl_wait();
  float* row = v + blockIdx.y * ld;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
    const float a = fmaxf(row[i], 0.f);
    row[i] = a * a;
  }
}

__global__ void ll_softcap_kernel(float* __restrict__ v, long long ld, int n, float cap) {
  pdl_wait();
  float* row = v + blockIdx.y * ld;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) row[i] = cap * tanhf(row[i] / cap);
}

// 64 x 64 tile, 16-deep steps, 256 threads of 4 x 4 outputs; plain fused multiply-adds in fp32.
__global__ void __launch_bounds__(256) ll_gemm_f32_kernel(const float* __restrict__ A, long long lda, const float* __restrict__ B,
                                                          long long ldb, float* __restrict__ C, long long ldc, int M, int N, int K) {
  pdl_wait();
  __shared__ float sA[16][68], sB[16][68];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
    if (k0 + lk < K) {
      if (m0 + lr < M) a = *reinterpret_cast<const float4*>(A + (long long)(m0 + lr) * lda + k0 + lk);
      if (n0 + lr < N) b = *reinterpret_cast<const float4*>(B + (long long)(n0 + lr) * ldb + k0 + lk);
    }
    __syncthreads();
    sA[lk][lr] = a.x; sA[lk + 1][lr] = a.y; sA[lk + 2][lr] = a.z; sA[lk + 3][lr] = a.w;
    sB[lk][lr] = b.x; sB[lk + 1][lr] = b.y; sB[lk + 2][lr] = b.z; sB[lk + 3][lr] = b.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&sA[k][ty * 4]);
      const float4 bv = *reinterpret_cast<const float4*>(&sB[k][tx * 4]);
      const float aa[4] = {av.x, av.y, av.z, av.w}, bb[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += aa[i] * bb[j];
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) C[(long long)m * ldc + n] = acc[i][j];
    }
  }
}

__global__ void ll_swiglu_f32_kernel(const float* __restrict__ gu, long long ld, float* __restrict__ act, long long lda, int E) {
  pdl_wait();
  const long long r = blockIdx.y;
  for (int j = blockIdx.x * blockDim.x + threadIdx.x; j < E; j += gridDim.x * blockDim.x) {
    const long long c = (long long)(j >> 6) * 128 + (j & 63);
    act[r * lda + j] = ll_silu(gu[r * ld + c]) * gu[r * ld + c + 64];
  }
}

__global__ void ll_advance_kernel(gb_seq_state* __restrict__ st, int* __restrict__ pos_out, int B, int n) {
  pdl_wait();
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  if (b >= B) return;
  const int p = st[b].abs_pos + n;
  st[b].abs_pos = p;
  st[b].cache_len = p;
  pos_out[b] = p;
}

}  // namespace gb

using namespace gb;

extern "C" int gb_ll_embed(const int* ids, const void* table, long long ld_table, int vocab, float* x, void* x16, long long ld16,
                           int rows, int d, int dtype, cudaStream_t st) {
  if (!ids || !table || !x || !x16 || rows <= 0 || d <= 0 || ld16 < d || vocab <= 0) return -1;
  if (dtype == 1)
    GB_PDL_LAUNCH(ll_embed_kernel<__nv_bfloat16>, dim3(rows), dim3(128), st, ids, (const __nv_bfloat16*)table, ld_table, vocab, x,
                  (__nv_bfloat16*)x16, ld16, rows, d);
  else if (dtype == 2)
    GB_PDL_LAUNCH(ll_embed_kernel<float>, dim3(rows), dim3(128), st, ids, (const float*)table, ld_table, vocab, x, (float*)x16, ld16, rows, d);
  else return -2;
  return gb_launch_rc();
}

extern "C" int gb_ll_postnorm(const float* y, long long ldy, const float* x, const float* w, float eps, float* x_out, void* x16,
                              long long ld16, int rows, int d, int dtype, cudaStream_t st) {
  if (!y || !x || !w || !x_out || rows <= 0 || d <= 0) return -1;
  const bool vec = d % 4 == 0 && ldy % 4 == 0 && ld16 % 4 == 0;
  const dim3 grid((rows + 7) / 8);
#define PN(T, V) GB_PDL_LAUNCH((ll_postnorm_kernel<T, V>), grid, dim3(256), st, y, ldy, x, w, eps, x_out, (T*)x16, ld16, rows, d)
  if (dtype == 1) { if (vec) PN(__nv_bfloat16, true); else PN(__nv_bfloat16, false); }
  else if (dtype == 2) { if (vec) PN(float, true); else PN(float, false); }
  else return -2;
#undef PN
  return gb_launch_rc();
}

extern "C" int gb_ll_norm_rows(const float* x, const int* row_idx, const float* w, float eps, void* out, long long ldo, int rows,
                               int d, int dtype, cudaStream_t st) {
  if (!x || !w || !out || rows <= 0 || d <= 0 || ldo < d) return -1;
  const dim3 grid((rows + 7) / 8);
  if (dtype == 1) GB_PDL_LAUNCH(ll_norm_rows_kernel<__nv_bfloat16>, grid, dim3(256), st, x, row_idx, w, eps, (__nv_bfloat16*)out, ldo, rows, d);
  else if (dtype == 2) GB_PDL_LAUNCH(ll_norm_rows_kernel<float>, grid, dim3(256), st, x, row_idx, w, eps, (float*)out, ldo, rows, d);
  else return -2;
  return gb_launch_rc();
}

// a warp per row while the row fits its registers, else a block per row
#define LL_ROWS(KERN, T, ...)                                                                                                 \
  do {                                                                                                                       \
    if (d <= 1024) {                                                                                                         \
      if (vec) GB_PDL_LAUNCH((KERN<T, 32, 4>), dim3((rows + 7) / 8), dim3(256), st, __VA_ARGS__);                               \
      else GB_PDL_LAUNCH((KERN<T, 32, 1>), dim3((rows + 7) / 8), dim3(256), st, __VA_ARGS__);                                   \
    } else if (vec) GB_PDL_LAUNCH((KERN<T, 256, 4>), dim3(rows), dim3(256), st, __VA_ARGS__);                                   \
    else GB_PDL_LAUNCH((KERN<T, 256, 1>), dim3(rows), dim3(256), st, __VA_ARGS__);                                              \
  } while (0)

static bool ll_norm_ok(int mode, const float* w) { return w && (mode == GB_LL_NORM_RMS || mode == GB_LL_NORM_LAYER); }
static uintptr_t ll_bits(const void* p) { return reinterpret_cast<uintptr_t>(p); }

extern "C" int gb_ll_embed_norm(const int* ids, const void* table, long long ld_table, int vocab, int mode, const float* w, const float* b,
                                float eps, float* x, int rows, int d, int dtype, cudaStream_t st) {
  if (!ids || !table || !x || rows <= 0 || d <= 0 || ld_table < d || vocab <= 0 || !ll_norm_ok(mode, w)) return -1;
  const bool vec = d % 4 == 0 && ld_table % 4 == 0 && ((ll_bits(table) | ll_bits(x)) & 15) == 0;
#define EN(T) LL_ROWS(ll_embed_norm_kernel, T, ids, (const T*)table, ld_table, vocab, mode, w, b, eps, x, rows, d)
  if (dtype == 1) EN(__nv_bfloat16);
  else if (dtype == 2) EN(float);
  else return -2;
#undef EN
  return gb_launch_rc();
}

extern "C" int gb_ll_add_norm(const float* y, long long ldy, float alpha, const float* x, const float* x0, const int* row_idx, int mode,
                              const float* w, const float* b, float eps, float* x_out, void* out, long long ldo, int rows, int d,
                              int dtype, cudaStream_t st) {
  if (!x || rows <= 0 || d <= 0 || (!x_out && !out) || (out && (!ll_norm_ok(mode, w) || ldo < d))) return -1;
  if (row_idx && (y || x0 || x_out)) return -3;
  const bool vec = d % 4 == 0 && (!y || ldy % 4 == 0) && (!out || ldo % 4 == 0) &&
                   ((ll_bits(y) | ll_bits(x) | ll_bits(x0) | ll_bits(x_out) | ll_bits(out)) & 15) == 0;
#define AN(T) LL_ROWS(ll_add_norm_kernel, T, y, ldy, alpha, x, x0, row_idx, mode, w, b, eps, x_out, (T*)out, ldo, rows, d)
  if (dtype == 1) AN(__nv_bfloat16);
  else if (dtype == 2) AN(float);
  else return -2;
#undef AN
  return gb_launch_rc();
}

extern "C" int gb_ll_relu2_f32(float* v, long long ld, int rows, int n, cudaStream_t st) {
  if (!v || rows <= 0 || n <= 0) return -1;
  GB_PDL_LAUNCH(ll_relu2_kernel, dim3((n + 1023) / 1024, rows), dim3(256), st, v, ld, n);
  return gb_launch_rc();
}

extern "C" int gb_ll_softcap(float* v, long long ld, int rows, int n, float cap, cudaStream_t st) {
  if (!v || rows <= 0 || n <= 0 || !(cap > 0.f)) return -1;
  GB_PDL_LAUNCH(ll_softcap_kernel, dim3((n + 1023) / 1024, rows), dim3(256), st, v, ld, n, cap);
  return gb_launch_rc();
}

extern "C" int gb_ll_gemm_f32(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc, int M, int N,
                              int K, cudaStream_t st) {
  if (!A || !B || !C || M <= 0 || N <= 0 || K <= 0 || K % 4 || lda % 4 || ldb % 4) return -1;
  GB_PDL_LAUNCH(ll_gemm_f32_kernel, dim3((N + 63) / 64, (M + 63) / 64), dim3(256), st, A, lda, B, ldb, C, ldc, M, N, K);
  return gb_launch_rc();
}

extern "C" int gb_ll_swiglu_f32(const float* gu, long long ld, float* act, long long lda, int rows, int E, cudaStream_t st) {
  if (!gu || !act || rows <= 0 || E <= 0 || E % 64) return -1;
  GB_PDL_LAUNCH(ll_swiglu_f32_kernel, dim3((E + 255) / 256, rows), dim3(256), st, gu, ld, act, lda, E);
  return gb_launch_rc();
}

extern "C" int gb_ll_advance(gb_seq_state* state, int* pos_out, int B, int n, cudaStream_t st) {
  if (!state || !pos_out || B <= 0 || n <= 0) return -1;
  GB_PDL_LAUNCH(ll_advance_kernel, dim3((B + 63) / 64), dim3(64), st, state, pos_out, B, n);
  return gb_launch_rc();
}
