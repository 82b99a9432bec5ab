// Token-step matrix-vector products of layer-list models (contract in gb_layers.h).  One token is bound by weight bytes
// and by the number of dependent launches, so what lies between two products (residual add with the norm of the
// sublayer's output, gated group norm, final norm) is the prologue of the second one: every block makes the input
// vector it needs in shared memory, and one block writes the new residual for the kernels after it.
#include <type_traits>

#include "sm100_common.cuh"
#include "gb_layers.h"
#include "decode_fmt.cuh"
#include "layers_util.cuh"

namespace gb {

constexpr int LV_WARPS = 8;
constexpr int LV_THREADS = LV_WARPS * 32;

__device__ __forceinline__ float ll_dot8(const float (&w)[8], const __nv_bfloat16* x) {
  const uint4 q = *reinterpret_cast<const uint4*>(x);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&q);
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); s += w[2 * i] * f.x + w[2 * i + 1] * f.y; }
  return s;
}
__device__ __forceinline__ float ll_dot8(const float (&w)[8], const float* x) {
  const float4 a = reinterpret_cast<const float4*>(x)[0], b = reinterpret_cast<const float4*>(x)[1];
  return w[0] * a.x + w[1] * a.y + w[2] * a.z + w[3] * a.w + w[4] * b.x + w[5] * b.y + w[6] * b.z + w[7] * b.w;
}

// sum over the block's 8 warps; every thread gets it.  `red` is 8 floats, reusable after the next block barrier.
__device__ __forceinline__ float ll_block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < LV_WARPS; ++i) t += red[i];
  return t;
}

struct LlGemv {
  const uint8_t* W; long long row_bytes; int N, K, B, d;
  const void* x16; long long ldx;
  const float* x; const float* y; long long ldy; const float* w1; const float* w2; float eps; float* x_out;
  const void* y16; long long ldy16; const void* z16; long long ldz; int parts;
  void* out; long long ldo; int out_f32; float softcap;
};

// Input vector of sequence b into xs[0, K).
template <int PRO, typename XT>
__device__ __forceinline__ void ll_prologue(const LlGemv& a, int b, XT* __restrict__ xs, float* red) {
  const int tid = threadIdx.x, d = a.d;
  if constexpr (PRO == 1) {
    const float* xr = a.x + (long long)b * d;
    constexpr int KEEP = 16;                       // values per thread kept in registers (d up to 4096)
    float v[KEEP];
    if (a.y) {
      const float* yr = a.y + b * a.ldy;
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        v[k] = i < d ? yr[i] : 0.f;
        ss += v[k] * v[k];
      }
      for (int i = tid + KEEP * LV_THREADS; i < d; i += LV_THREADS) ss += yr[i] * yr[i];
      const float inv = ll_inv_rms(ll_block_sum(ss, red), d, a.eps);
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        if (i < d) v[k] = xr[i] + v[k] * inv * a.w1[i];
      }
      for (int i = tid; i < d; i += LV_THREADS) {
        const int k = (i - tid) / LV_THREADS;
        if (k >= KEEP) {
          const float o = xr[i] + yr[i] * inv * a.w1[i];
          if (blockIdx.x == 0 && a.x_out) a.x_out[(long long)b * d + i] = o;
          if (!a.w2) xs[i] = Cvt<XT>::from_f(o);
        }
      }
    } else {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        v[k] = i < d ? xr[i] : 0.f;
      }
      for (int i = tid + KEEP * LV_THREADS; i < d; i += LV_THREADS) {
        if (blockIdx.x == 0 && a.x_out) a.x_out[(long long)b * d + i] = xr[i];
        if (!a.w2) xs[i] = Cvt<XT>::from_f(xr[i]);
      }
    }
    if (blockIdx.x == 0 && a.x_out) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        if (i < d) a.x_out[(long long)b * d + i] = v[k];
      }
    }
    if (a.w2) {                                    // the model's last norm on top (host: d <= KEEP * LV_THREADS)
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        if (i < d) ss += v[k] * v[k];
      }
      const float inv = ll_inv_rms(ll_block_sum(ss, red), d, a.eps);
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        if (i < d) v[k] = v[k] * inv * a.w2[i];
      }
    }
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = tid + k * LV_THREADS;
      if (i < d) xs[i] = Cvt<XT>::from_f(v[k]);
    }
  } else {                                         // PRO == 2: gated norm in equal parts, one warp per part
    const XT* yr = reinterpret_cast<const XT*>(a.y16) + b * a.ldy16;
    const XT* zr = reinterpret_cast<const XT*>(a.z16) + b * a.ldz;
    const int per = d / a.parts, warp = tid >> 5, lane = tid & 31;
    if (a.parts >= LV_WARPS) {
      for (int p = warp; p < a.parts; p += LV_WARPS) {
        float ss = 0.f;
        for (int i = lane; i < per; i += 32) {
          const float v = Cvt<XT>::to_f(yr[p * per + i]) * ll_silu(Cvt<XT>::to_f(zr[p * per + i]));
          ss += v * v;
        }
        const float inv = ll_inv_rms(warp_sum(ss), per, a.eps);
        for (int i = lane; i < per; i += 32) {
          const float v = Cvt<XT>::to_f(yr[p * per + i]) * ll_silu(Cvt<XT>::to_f(zr[p * per + i]));
          xs[p * per + i] = Cvt<XT>::from_f(v * inv * a.w1[p * per + i]);
        }
      }
    } else {
      for (int p = 0; p < a.parts; ++p) {          // few parts: the whole block works on each
        constexpr int KEEP = 8;
        float v[KEEP];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
          const int i = tid + k * LV_THREADS;
          v[k] = i < per ? Cvt<XT>::to_f(yr[p * per + i]) * ll_silu(Cvt<XT>::to_f(zr[p * per + i])) : 0.f;
          ss += v[k] * v[k];
        }
        for (int i = tid + KEEP * LV_THREADS; i < per; i += LV_THREADS) {
          const float t = Cvt<XT>::to_f(yr[p * per + i]) * ll_silu(Cvt<XT>::to_f(zr[p * per + i]));
          ss += t * t;
        }
        const float inv = ll_inv_rms(ll_block_sum(ss, red), per, a.eps);
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
          const int i = tid + k * LV_THREADS;
          if (i < per) xs[p * per + i] = Cvt<XT>::from_f(v[k] * inv * a.w1[p * per + i]);
        }
        for (int i = tid + KEEP * LV_THREADS; i < per; i += LV_THREADS) {
          const float t = Cvt<XT>::to_f(yr[p * per + i]) * ll_silu(Cvt<XT>::to_f(zr[p * per + i]));
          xs[p * per + i] = Cvt<XT>::from_f(t * inv * a.w1[p * per + i]);
        }
      }
    }
  }
  for (int i = d + tid; i < a.K; i += LV_THREADS) xs[i] = Cvt<XT>::from_f(0.f);
}

template <int FMT, int NB, int KS, typename XT>
__device__ __forceinline__ void ll_row(const uint8_t* __restrict__ wrow, int K, const XT* x, long long ldx, int nb, int ks,
                                       float (&acc)[NB]) {
  const int lane = threadIdx.x & 31;
#pragma unroll 4
  for (int u = lane + 32 * ks; u < (K >> 3); u += 32 * KS) {
    float w[8];
    load8<FMT>(wrow, u, w);
#pragma unroll
    for (int j = 0; j < NB; ++j)
      if (j < nb) acc[j] += ll_dot8(w, x + j * ldx + 8 * u);
  }
}

// KS warps share a stored row (short rows spread over more of the machine); NB sequences per pass over the row.
template <int FMT, typename XT, int PRO, int SWI, int NB, int KS>
__global__ void __launch_bounds__(LV_THREADS) ll_gemv_kernel(const __grid_constant__ LlGemv a) {
  pdl_wait();
  extern __shared__ __align__(16) uint8_t lv_dyn[];
  __shared__ float red[LV_WARPS];
  __shared__ float part[2][LV_WARPS][NB];
  XT* xs = reinterpret_cast<XT*>(lv_dyn);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ric = warp / KS, ks = warp % KS;
  const XT* xin = reinterpret_cast<const XT*>(a.x16);
  long long ldx = a.ldx;
  if constexpr (PRO != 0) {
    for (int b = 0; b < a.B; ++b) ll_prologue<PRO, XT>(a, b, xs + (long long)b * a.K, red);
    __syncthreads();
    xin = xs;
    ldx = a.K;
  }
  const int n_out = SWI ? a.N / 2 : a.N;
  const int j = blockIdx.x * (LV_WARPS / KS) + ric;
  const bool live = j < n_out;
  const long long row = SWI ? (long long)(j >> 6) * 128 + (j & 63) : j;
  const uint8_t* w0 = a.W + (live ? row : 0) * a.row_bytes;
  const uint8_t* w1 = w0 + 64 * a.row_bytes;
  for (int b0 = 0; b0 < a.B; b0 += NB) {
    const int nb = min(NB, a.B - b0);
    float acc[NB], acu[NB];
#pragma unroll
    for (int k = 0; k < NB; ++k) { acc[k] = 0.f; acu[k] = 0.f; }
    if (live) {
      ll_row<FMT, NB, KS, XT>(w0, a.K, xin + b0 * ldx, ldx, nb, ks, acc);
      if constexpr (SWI != 0) ll_row<FMT, NB, KS, XT>(w1, a.K, xin + b0 * ldx, ldx, nb, ks, acu);
    }
#pragma unroll
    for (int k = 0; k < NB; ++k) {
      acc[k] = warp_sum(acc[k]);
      if constexpr (SWI != 0) acu[k] = warp_sum(acu[k]);
    }
    if constexpr (KS > 1) {
      if (lane == 0) {
#pragma unroll
        for (int k = 0; k < NB; ++k) { part[0][warp][k] = acc[k]; part[1][warp][k] = acu[k]; }
      }
      __syncthreads();
      if (ks == 0) {
#pragma unroll
        for (int k = 0; k < NB; ++k) {
          acc[k] = 0.f; acu[k] = 0.f;
#pragma unroll
          for (int s = 0; s < KS; ++s) { acc[k] += part[0][ric * KS + s][k]; acu[k] += part[1][ric * KS + s][k]; }
        }
      }
      __syncthreads();
    }
    if (live && ks == 0 && lane == 0) {
#pragma unroll
      for (int k = 0; k < NB; ++k) {
        if (k >= nb) continue;
        float v = SWI ? ll_silu(acc[k]) * acu[k] : acc[k];
        if (a.softcap > 0.f) v = a.softcap * tanhf(v / a.softcap);
        if (a.out_f32) reinterpret_cast<float*>(a.out)[(long long)(b0 + k) * a.ldo + j] = v;
        else reinterpret_cast<XT*>(a.out)[(long long)(b0 + k) * a.ldo + j] = Cvt<XT>::from_f(v);
      }
    }
  }
}

template <int FMT, typename XT, int PRO, int SWI>
static int ll_gemv_go(const LlGemv& a, cudaStream_t st) {
  const size_t smem = PRO ? (size_t)a.B * a.K * sizeof(XT) : 0;
  if (smem > 200 * 1024) return -3;
  const int n_out = SWI ? a.N / 2 : a.N;
  const bool split = n_out <= 8192 && a.K >= 256;
#define GO(NB, KS) GB_PDL_LAUNCH_SMEM((ll_gemv_kernel<FMT, XT, PRO, SWI, NB, KS>), dim3((n_out + LV_WARPS / KS - 1) / (LV_WARPS / KS)), \
                                      dim3(LV_THREADS), smem, st, a)
  if (a.B == 1) { if (split) GO(1, 4); else GO(1, 1); }
  else { if (split) GO(4, 4); else GO(4, 1); }
#undef GO
  return gb_launch_rc();
}

template <int FMT, typename XT>
static int ll_gemv_pro(const LlGemv& a, int prologue, int swiglu, cudaStream_t st) {
  switch (prologue) {
    case 0: return swiglu ? ll_gemv_go<FMT, XT, 0, 1>(a, st) : ll_gemv_go<FMT, XT, 0, 0>(a, st);
    case 1: return swiglu ? ll_gemv_go<FMT, XT, 1, 1>(a, st) : ll_gemv_go<FMT, XT, 1, 0>(a, st);
    case 2: return swiglu ? -1 : ll_gemv_go<FMT, XT, 2, 0>(a, st);
  }
  return -1;
}

}  // namespace gb

using namespace gb;

extern "C" int gb_ll_gemv(const gb_ll_gemv_args* p, cudaStream_t st) {
  if (!p || !p->W || !p->out || p->N <= 0 || p->K <= 0 || p->B <= 0 || p->B > 8 || p->d <= 0 || p->d > p->K) return -1;
  const long long rb = p->K % 8 ? -1 : p->fmt == GB_W_BF16 ? 2LL * p->K : p->fmt == GB_W_F32 ? 4LL * p->K : -1;
  if (rb < 0 || (p->swiglu && p->N % 128)) return -1;
  if (p->prologue == 0 && (!p->x16 || p->ldx % 8)) return -1;
  if (p->prologue == 1 && (!p->x || (p->y && !p->w1) || (p->w2 && p->d > 4096))) return -1;
  if (p->prologue == 2 && (!p->y16 || !p->z16 || !p->w1 || p->parts <= 0 || p->d % p->parts)) return -1;
  LlGemv a{};
  a.W = static_cast<const uint8_t*>(p->W); a.row_bytes = rb; a.N = p->N; a.K = p->K; a.B = p->B; a.d = p->d;
  a.x16 = p->x16; a.ldx = p->ldx; a.x = p->x; a.y = p->y; a.ldy = p->ldy; a.w1 = p->w1; a.w2 = p->w2; a.eps = p->eps;
  a.x_out = p->x_out; a.y16 = p->y16; a.ldy16 = p->ldy16; a.z16 = p->z16; a.ldz = p->ldz; a.parts = p->parts;
  a.out = p->out; a.ldo = p->ldo; a.out_f32 = p->out_f32; a.softcap = p->softcap;
  if (p->dtype == 1 && p->fmt == GB_W_BF16) return ll_gemv_pro<GB_W_BF16, __nv_bfloat16>(a, p->prologue, p->swiglu, st);
  if (p->dtype == 2 && p->fmt == GB_W_F32) return ll_gemv_pro<GB_W_F32, float>(a, p->prologue, p->swiglu, st);
  return -2;
}
