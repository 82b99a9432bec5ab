// Token-step matrix-vector products of layer-list models (interface in gb_layers.h).  One token is bound by weight bytes
// and by the number of dependent launches, so what lies between two products (residual add with the norm of the
// sublayer's output, gated group norm, final norm) is the prologue of the second one: every block makes the input
// vector it needs in shared memory, and one block writes the new residual for the kernels after it.  Weights do not depend
// on the kernel before, so the first loads of a block's rows are issued ahead of the wait for it; a block walks several
// rows when there are many, with the next row's loads issued before the current row is reduced.
#include <type_traits>

#include "sm100_common.cuh"
#include "gb_layers.h"
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
  const float* v32; const float* sq; int n_sq;
  void* out; long long ldo; int out_f32; float softcap;
  const float* x0; float alpha; const float* b1; int norm_mode;
  int n1; void* out2; long long ldo2;
};

// Input vector of sequence b into xs[0, K).
template <int PRO, typename XT>
__device__ __forceinline__ void ll_prologue(const LlGemv& a, int b, XT* __restrict__ xs, float* red, float* part_inv) {
  const int tid = threadIdx.x, d = a.d;
  if constexpr (PRO == 1) {
    const float* xr = a.x + (long long)b * d;
    constexpr int KEEP = 16;                       // values per thread kept in registers (d up to 4096)
    float v[KEEP];
    const bool writes = blockIdx.x == 0 && a.x_out != nullptr;
    if (a.y) {
      const float* yr = a.y + b * a.ldy;
      float xv[KEEP];
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        v[k] = i < d ? yr[i] : 0.f;
        xv[k] = i < d ? xr[i] : 0.f;
        ss += v[k] * v[k];
      }
      for (int i = tid + KEEP * LV_THREADS; i < d; i += LV_THREADS) ss += yr[i] * yr[i];
      const float inv = ll_inv_rms(ll_block_sum(ss, red), d, a.eps);
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        if (i < d) v[k] = xv[k] + v[k] * inv * a.w1[i];
      }
      for (int i = tid + KEEP * LV_THREADS; i < d; i += LV_THREADS) {
        const float o = xr[i] + yr[i] * inv * a.w1[i];
        if (writes) a.x_out[(long long)b * d + i] = o;
        xs[i] = Cvt<XT>::from_f(o);
      }
    } else {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        v[k] = i < d ? xr[i] : 0.f;
      }
      for (int i = tid + KEEP * LV_THREADS; i < d; i += LV_THREADS) {
        if (writes) a.x_out[(long long)b * d + i] = xr[i];
        xs[i] = Cvt<XT>::from_f(xr[i]);
      }
    }
    if (writes) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = tid + k * LV_THREADS;
        if (i < d) a.x_out[(long long)b * d + i] = v[k];
      }
    }
    if (a.w2) {                                    // the model's last norm on top (host: d <= KEEP * LV_THREADS)
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < KEEP; ++k) ss += v[k] * v[k];      // values past d are zero
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
  } else if constexpr (PRO == 4) {                 // weighted RMS norm of a 16-bit (fp32) vector
    const XT* xr = reinterpret_cast<const XT*>(a.x16) + b * a.ldx;
    float ss = 0.f;
    for (int i = tid; i < d; i += LV_THREADS) { const float v = Cvt<XT>::to_f(xr[i]); ss += v * v; }
    const float inv = ll_inv_rms(ll_block_sum(ss, red), d, a.eps);
    for (int i = tid; i < d; i += LV_THREADS) xs[i] = Cvt<XT>::from_f(Cvt<XT>::to_f(xr[i]) * inv * a.w1[i]);
  } else if constexpr (PRO == 5) {                 // residual add, then the norm ahead of the sublayers
    const float* xr = a.x + (long long)b * d;
    const float* yr = a.y ? a.y + b * a.ldy : nullptr;
    const float* x0 = a.x0 ? a.x0 + (long long)b * d : nullptr;
    float* xo = blockIdx.x == 0 && a.x_out ? a.x_out + (long long)b * d : nullptr;
    constexpr int KEEP = 16;                       // values per thread kept in registers (d up to 4096); the rest is made again
    auto value = [&](int i) {
      float v = xr[i];
      if (yr) v += a.alpha * yr[i];
      if (x0) v += x0[i];
      return v;
    };
    float v[KEEP];
    float sum = 0.f, dev = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = tid + k * LV_THREADS;
      v[k] = i < d ? value(i) : 0.f;
      sum += v[k];
    }
    for (int i = tid + KEEP * LV_THREADS; i < d; i += LV_THREADS) sum += value(i);
    const float mean = a.norm_mode == GB_LL_NORM_LAYER ? ll_block_sum(sum, red) / (float)d : 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = tid + k * LV_THREADS;
      if (i < d) { const float c = v[k] - mean; dev += c * c; }
    }
    for (int i = tid + KEEP * LV_THREADS; i < d; i += LV_THREADS) { const float c = value(i) - mean; dev += c * c; }
    const float inv = ll_inv_rms(ll_block_sum(dev, red), d, a.eps);
    auto put = [&](int i, float u) {
      if (xo) xo[i] = u;
      xs[i] = Cvt<XT>::from_f((u - mean) * inv * a.w1[i] + (a.b1 ? a.b1[i] : 0.f));
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = tid + k * LV_THREADS;
      if (i < d) put(i, v[k]);
    }
    for (int i = tid + KEEP * LV_THREADS; i < d; i += LV_THREADS) put(i, value(i));
  } else if constexpr (PRO == 3) {                 // gated values and their sums of squares from the step kernel
    const float* vr = a.v32 + (long long)b * d;
    const float* sq = a.sq + (long long)b * a.n_sq;
    const int per = d / a.parts, nq = a.n_sq / a.parts, warp = tid >> 5, lane = tid & 31;
    for (int p = warp; p < a.parts; p += LV_WARPS) {
      float ss = 0.f;
      for (int i = lane; i < nq; i += 32) ss += sq[p * nq + i];
      ss = warp_sum(ss);
      if (lane == 0) part_inv[p] = ll_inv_rms(ss, per, a.eps);
    }
    __syncthreads();
#pragma unroll 4
    for (int i = tid; i < d; i += LV_THREADS) xs[i] = Cvt<XT>::from_f(vr[i] * part_inv[i / per] * a.w1[i]);
    __syncthreads();                               // part_inv is the next sequence's, too
  } else {                                         // PRO == 2: gated norm in equal parts, one warp per part
    const XT* yr = reinterpret_cast<const XT*>(a.y16) + b * a.ldy16;
    const XT* zr = reinterpret_cast<const XT*>(a.z16) + b * a.ldz;
    const int per = d / a.parts, warp = tid >> 5, lane = tid & 31;
    if (a.parts >= LV_WARPS) {
      for (int p = warp; p < a.parts; p += LV_WARPS) {
        float ss = 0.f;
        for (int i = lane; i < per; i += 32) {
          const float v = Cvt<XT>::to_f(yr[p * per + i]) * ll_silu_t<XT>(Cvt<XT>::to_f(zr[p * per + i]));
          ss += v * v;
        }
        const float inv = ll_inv_rms(warp_sum(ss), per, a.eps);
        for (int i = lane; i < per; i += 32) {
          const float v = Cvt<XT>::to_f(yr[p * per + i]) * ll_silu_t<XT>(Cvt<XT>::to_f(zr[p * per + i]));
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
          v[k] = i < per ? Cvt<XT>::to_f(yr[p * per + i]) * ll_silu_t<XT>(Cvt<XT>::to_f(zr[p * per + i])) : 0.f;
          ss += v[k] * v[k];
        }
        for (int i = tid + KEEP * LV_THREADS; i < per; i += LV_THREADS) {
          const float t = Cvt<XT>::to_f(yr[p * per + i]) * ll_silu_t<XT>(Cvt<XT>::to_f(zr[p * per + i]));
          ss += t * t;
        }
        const float inv = ll_inv_rms(ll_block_sum(ss, red), per, a.eps);
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
          const int i = tid + k * LV_THREADS;
          if (i < per) xs[p * per + i] = Cvt<XT>::from_f(v[k] * inv * a.w1[p * per + i]);
        }
        for (int i = tid + KEEP * LV_THREADS; i < per; i += LV_THREADS) {
          const float t = Cvt<XT>::to_f(yr[p * per + i]) * ll_silu_t<XT>(Cvt<XT>::to_f(zr[p * per + i]));
          xs[p * per + i] = Cvt<XT>::from_f(t * inv * a.w1[p * per + i]);
        }
      }
    }
  }
  for (int i = d + tid; i < a.K; i += LV_THREADS) xs[i] = Cvt<XT>::from_f(0.f);
}

// Raw stored values of one 8-value unit.
template <int FMT> struct LlRaw;
template <> struct LlRaw<GB_W_BF16> {
  uint4 q;
  __device__ __forceinline__ void load(const uint8_t* row, int u) { q = __ldg(reinterpret_cast<const uint4*>(row) + u); }
  __device__ __forceinline__ void expand(float (&w)[8]) const {
    const uint32_t v[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = Cvt<__nv_bfloat16>::unpack2(v[i]); w[2 * i] = f.x; w[2 * i + 1] = f.y; }
  }
};
template <> struct LlRaw<GB_W_F32> {
  float4 a, b;
  __device__ __forceinline__ void load(const uint8_t* row, int u) {
    a = __ldg(reinterpret_cast<const float4*>(row) + 2 * u);
    b = __ldg(reinterpret_cast<const float4*>(row) + 2 * u + 1);
  }
  __device__ __forceinline__ void expand(float (&w)[8]) const {
    w[0] = a.x; w[1] = a.y; w[2] = a.z; w[3] = a.w; w[4] = b.x; w[5] = b.y; w[6] = b.z; w[7] = b.w;
  }
};

template <int FMT, int NB, typename XT>
__device__ __forceinline__ void ll_accum(const LlRaw<FMT>& raw, int u, const XT* x, long long ldx, int nb, float (&acc)[NB]) {
  float w[8];
  raw.expand(w);
#pragma unroll
  for (int j = 0; j < NB; ++j)
    if (j < nb) acc[j] += ll_dot8(w, x + j * ldx + 8 * u);
}

// KS warps share a stored row (short rows spread over more of the machine); NB sequences per pass over the row.
template <int FMT, typename XT, int PRO, int SWI, int NB, int KS>
__global__ void __launch_bounds__(LV_THREADS) ll_gemv_kernel(const __grid_constant__ LlGemv a) {
  constexpr int PF = (SWI ? 4 : 8) / (FMT == GB_W_F32 ? 2 : 1);      // units per lane and row that are loaded ahead
  extern __shared__ __align__(16) uint8_t lv_dyn[];
  __shared__ float red[LV_WARPS];
  __shared__ float part_inv[PRO == 3 ? 256 : 1];
  __shared__ float part[2][LV_WARPS][NB];
  XT* xs = reinterpret_cast<XT*>(lv_dyn);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ric = warp / KS, ks = warp % KS;
  const int n_out = SWI ? a.N / 2 : a.N, units = a.K >> 3, u0 = lane + 32 * ks;
  constexpr int RPB = LV_WARPS / KS, US = 32 * KS;
  auto row_of = [&](int j) { return a.W + (SWI ? (long long)(j >> 6) * 128 + (j & 63) : (long long)j) * a.row_bytes; };
  LlRaw<FMT> g[PF], up[SWI ? PF : 1];
  auto fetch = [&](int j) {
    if (j >= n_out) return;
    const uint8_t* w = row_of(j);
#pragma unroll
    for (int k = 0; k < PF; ++k)
      if (u0 + k * US < units) {
        g[k].load(w, u0 + k * US);
        if constexpr (SWI != 0) up[k].load(w + 64 * a.row_bytes, u0 + k * US);
      }
  };
  fetch(blockIdx.x * RPB + ric);
  pdl_wait();
  const XT* xin = reinterpret_cast<const XT*>(a.x16);
  long long ldx = a.ldx;
  if constexpr (PRO != 0) {
    for (int b = 0; b < a.B; ++b) ll_prologue<PRO, XT>(a, b, xs + (long long)b * a.K, red, part_inv);
    __syncthreads();
    xin = xs;
    ldx = a.K;
  }
  // every warp of the block makes the same number of trips: rows past the end still take part in the barriers
  for (int j0 = blockIdx.x * RPB; j0 < n_out; j0 += gridDim.x * RPB) {
    const int j = j0 + ric;
    const bool live = j < n_out;
    for (int b0 = 0; b0 < a.B; b0 += NB) {
      const int nb = min(NB, a.B - b0);
      float acc[NB], acu[NB];
#pragma unroll
      for (int k = 0; k < NB; ++k) { acc[k] = 0.f; acu[k] = 0.f; }
      if (live) {
        if (b0 > 0) fetch(j);
        const XT* xb = xin + b0 * ldx;
#pragma unroll
        for (int k = 0; k < PF; ++k)
          if (u0 + k * US < units) {
            ll_accum<FMT, NB, XT>(g[k], u0 + k * US, xb, ldx, nb, acc);
            if constexpr (SWI != 0) ll_accum<FMT, NB, XT>(up[k], u0 + k * US, xb, ldx, nb, acu);
          }
        const uint8_t* w = row_of(j);
#pragma unroll 4
        for (int u = u0 + PF * US; u < units; u += US) {
          LlRaw<FMT> r0, r1;
          r0.load(w, u);
          if constexpr (SWI != 0) r1.load(w + 64 * a.row_bytes, u);
          ll_accum<FMT, NB, XT>(r0, u, xb, ldx, nb, acc);
          if constexpr (SWI != 0) ll_accum<FMT, NB, XT>(r1, u, xb, ldx, nb, acu);
        }
      }
      if (b0 + NB >= a.B) fetch(j + gridDim.x * RPB);
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
          if (a.n1 > 0 && j >= a.n1) {
            v = fmaxf(v, 0.f);
            reinterpret_cast<XT*>(a.out2)[(long long)(b0 + k) * a.ldo2 + j - a.n1] = Cvt<XT>::from_f(v * v);
          } else if (a.out_f32) reinterpret_cast<float*>(a.out)[(long long)(b0 + k) * a.ldo + j] = v;
          else reinterpret_cast<XT*>(a.out)[(long long)(b0 + k) * a.ldo + j] = Cvt<XT>::from_f(v);
        }
      }
    }
  }
}

template <int FMT, typename XT, int PRO, int SWI>
static int ll_gemv_go(const LlGemv& a, cudaStream_t st) {
  const size_t smem = PRO ? (size_t)a.B * a.K * sizeof(XT) : 0;
  if (smem > 200 * 1024) return -3;
  const int n_out = SWI ? a.N / 2 : a.N;
  // warps per row: enough of them to keep loads in flight on every SM, more for long rows
  const int units = a.K >> 3;
  const int ks = (n_out < 148 * 16 || units > 512) ? 4 : (n_out < 148 * 64 || units > 256) ? 2 : 1;
  // blocks: what is resident at once, and then so many that all of them make the same number of trips
#define GO(NB, KS)                                                                                                                 \
  do {                                                                                                                             \
    auto kern = ll_gemv_kernel<FMT, XT, PRO, SWI, NB, KS>;                                                                         \
    static int occ = 0;                                                                                                            \
    if (!occ && (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&occ, kern, LV_THREADS, 16 * 1024) != cudaSuccess || occ < 1)) occ = 2; \
    const int groups = (n_out + LV_WARPS / KS - 1) / (LV_WARPS / KS), trips = (groups + 148 * occ - 1) / (148 * occ);              \
    GB_PDL_LAUNCH_SMEM(kern, dim3((groups + trips - 1) / trips), dim3(LV_THREADS), smem, st, a);                                   \
  } while (0)
#define GOK(NB) do { if (ks == 4) GO(NB, 4); else if (ks == 2) GO(NB, 2); else GO(NB, 1); } while (0)
  if (a.B == 1) GOK(1);
  else GOK(4);
#undef GOK
#undef GO
  return gb_launch_rc();
}

template <int FMT, typename XT>
static int ll_gemv_pro(const LlGemv& a, int prologue, int swiglu, cudaStream_t st) {
  switch (prologue) {
    case 0: return swiglu ? ll_gemv_go<FMT, XT, 0, 1>(a, st) : ll_gemv_go<FMT, XT, 0, 0>(a, st);
    case 1: return swiglu ? ll_gemv_go<FMT, XT, 1, 1>(a, st) : ll_gemv_go<FMT, XT, 1, 0>(a, st);
    case 2: return swiglu ? -1 : ll_gemv_go<FMT, XT, 2, 0>(a, st);
    case 3: return swiglu ? -1 : ll_gemv_go<FMT, XT, 3, 0>(a, st);
    case 4: return swiglu ? -1 : ll_gemv_go<FMT, XT, 4, 0>(a, st);
    case 5: return swiglu ? -1 : ll_gemv_go<FMT, XT, 5, 0>(a, st);
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
  if (p->prologue == 3 && (!p->v32 || !p->sq || !p->w1 || p->parts <= 0 || p->parts > 256 || p->d % p->parts || p->n_sq <= 0 || p->n_sq % p->parts)) return -1;
  if (p->prologue == 4 && (!p->x16 || !p->w1)) return -1;
  if (p->prologue == 5 && (!p->x || !p->w1 || (p->x_out && (p->x_out == p->x || p->x_out == p->x0)))) return -1;
  if (p->n1 > 0 && (p->swiglu || !p->out2 || p->n1 > p->N)) return -1;
  LlGemv a{};
  a.x0 = p->x0; a.alpha = p->alpha; a.b1 = p->b1; a.norm_mode = p->norm_mode;
  a.n1 = p->n1; a.out2 = p->out2; a.ldo2 = p->ldo2;
  a.v32 = p->v32; a.sq = p->sq; a.n_sq = p->n_sq;
  a.W = static_cast<const uint8_t*>(p->W); a.row_bytes = rb; a.N = p->N; a.K = p->K; a.B = p->B; a.d = p->d;
  a.x16 = p->x16; a.ldx = p->ldx; a.x = p->x; a.y = p->y; a.ldy = p->ldy; a.w1 = p->w1; a.w2 = p->w2; a.eps = p->eps;
  a.x_out = p->x_out; a.y16 = p->y16; a.ldy16 = p->ldy16; a.z16 = p->z16; a.ldz = p->ldz; a.parts = p->parts;
  a.out = p->out; a.ldo = p->ldo; a.out_f32 = p->out_f32; a.softcap = p->softcap;
  if (p->dtype == 1 && p->fmt == GB_W_BF16) return ll_gemv_pro<GB_W_BF16, __nv_bfloat16>(a, p->prologue, p->swiglu, st);
  if (p->dtype == 2 && p->fmt == GB_W_F32) return ll_gemv_pro<GB_W_F32, float>(a, p->prologue, p->swiglu, st);
  return -2;
}
