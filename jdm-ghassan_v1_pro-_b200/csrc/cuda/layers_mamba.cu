// Mamba-2 mixer of layer-list models (interface in gb_layers.h): causal convolution with its carried inputs, the state
// recurrence token by token (fp32 for every size; the chunked tensor-core form is in layers_ssd.cu), the gated group
// norm, and the one-token step that fuses convolution and recurrence.
//
// Nothing has to be cleared when a sequence slot is used again: inputs before position 0 count as zero and the state
// starts at zero when the first new token is at position 0.
#include <type_traits>

#include "sm100_common.cuh"
#include "gb_layers.h"
#include "layers_util.cuh"

namespace gb {

constexpr int CONV_TT = 32;      // tokens per thread

// Input of channel c at position p0 + t (t < 0: from the carried rows).
template <typename T>
__device__ __forceinline__ float ll_conv_in(const gb_ll_mamba_args& a, const T* proj_b, const T* ring, int p0, int t, int c, int C) {
  if (t >= 0) return Cvt<T>::to_f(proj_b[t * a.ld_proj + c]);
  const int p = p0 + t;
  return p < 0 ? 0.f : Cvt<T>::to_f(ring[(long long)(p % a.taps) * C + c]);
}

template <typename T>
__device__ __forceinline__ void ll_conv_out(const gb_ll_mamba_args& a, long long row, int c, float v) {
  const int n = a.H * a.P, gn = a.G * a.N;
  if (c < n) {
    const int h = c / a.P;
    reinterpret_cast<T*>(a.xh)[(row * a.H + h) * a.Pp + (c - h * a.P)] = Cvt<T>::from_f(v);
  } else {
    const bool is_b = c < n + gn;
    const int e = c - n - (is_b ? 0 : gn), g = e / a.N;
    reinterpret_cast<T*>(is_b ? a.bc : a.cc)[(row * a.G + g) * a.Np + (e - g * a.N)] = Cvt<T>::from_f(v);
  }
}

// grid (channels / 128, token tiles, B); thread = channel.  MAXT: taps held in registers.
template <typename T, int MAXT>
__global__ void __launch_bounds__(128) ll_conv_kernel(const __grid_constant__ gb_ll_mamba_args a) {
  pdl_wait();
  const int n = a.H * a.P, C = n + 2 * a.G * a.N;
  const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.z, t0 = blockIdx.y * CONV_TT;
  if (c >= C) return;
  const int p0 = a.st[b].abs_pos;
  const T* proj = reinterpret_cast<const T*>(a.proj) + (long long)b * a.n * a.ld_proj + n;
  T* ring = reinterpret_cast<T*>(a.conv_state) + (long long)b * a.taps * C;
  const float* kw = a.conv_w + (long long)c * a.taps;
  const float bias = a.conv_b[c];
  const int t1 = min(a.n, t0 + CONV_TT);
  float w[MAXT], x[MAXT];        // x[k]: input k + 1 tokens before the current one
#pragma unroll
  for (int k = 0; k < MAXT; ++k) {
    w[k] = k < a.taps ? kw[a.taps - 1 - k] : 0.f;      // w[0] belongs to the current token
    x[k] = k < a.taps - 1 ? ll_conv_in<T>(a, proj, ring, p0, t0 - 1 - k, c, C) : 0.f;
  }
  for (int t = t0; t < t1; ++t) {
    const float cur = Cvt<T>::to_f(proj[t * a.ld_proj + c]);
    float s = bias + w[0] * cur;
#pragma unroll
    for (int k = 1; k < MAXT; ++k) s += w[k] * x[k - 1];
    ll_conv_out<T>(a, (long long)b * a.n + t, c, ll_silu_t<T>(s));
#pragma unroll
    for (int k = MAXT - 1; k > 0; --k) x[k] = x[k - 1];
    x[0] = cur;
  }
  // The block of the first tile is the only reader of this channel's carried inputs, so it also replaces them.
  if (t0 == 0)
    for (int t = max(0, a.n - a.taps); t < a.n; ++t) ring[(long long)((p0 + t) % a.taps) * C + c] = proj[t * a.ld_proj + c];
}

// Four channels per thread (sizes and pitches in multiples of four), `tile` tokens: one vector load and store per token, the
// inputs of the last taps - 1 tokens in registers, four tokens' loads ahead of their use.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) ll_conv_vec_kernel(const __grid_constant__ gb_ll_mamba_args a, int tile) {
  pdl_wait();
  const int n = a.H * a.P, gn = a.G * a.N, C = n + 2 * gn;
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4, b = blockIdx.z, t0 = blockIdx.y * tile, t1 = min(a.n, t0 + tile);
  if (c >= C) return;
  constexpr int PF = 4;
  const T* src = reinterpret_cast<const T*>(a.proj) + (long long)b * a.n * a.ld_proj + n + c;
  LlRaw4<T> in[PF];
#pragma unroll
  for (int u = 0; u < PF; ++u)
    if (t0 + u < t1) in[u].load(src + (t0 + u) * a.ld_proj);
  const int p0 = a.st[b].abs_pos;
  T* ring = reinterpret_cast<T*>(a.conv_state) + (long long)b * TAPS * C + c;
  float w[TAPS][4], x[TAPS][4], bias[4];     // x[k]: inputs k + 1 tokens before the current one
#pragma unroll
  for (int e = 0; e < 4; ++e) bias[e] = a.conv_b[c + e];
  {
    float f[TAPS][4];                        // the taps of four channels are consecutive
#pragma unroll
    for (int i = 0; i < TAPS; ++i) { LlRaw4<float> r; r.load(a.conv_w + (long long)c * TAPS + 4 * i); r.expand(f[i]); }
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int k = 0; k < TAPS; ++k) { const int i = e * TAPS + TAPS - 1 - k; w[k][e] = f[i >> 2][i & 3]; }
  }
#pragma unroll
  for (int k = 1; k < TAPS; ++k) {
    const int t = t0 - k;
    LlRaw4<T> r;
    if (t >= 0) { r.load(src + t * a.ld_proj); r.expand(x[k - 1]); }
    else if (p0 + t >= 0) { r.load(ring + (long long)((p0 + t) % TAPS) * C); r.expand(x[k - 1]); }
    else {
#pragma unroll
      for (int e = 0; e < 4; ++e) x[k - 1][e] = 0.f;
    }
  }
  T* dst;
  long long step;
  if (c < n) {
    const int h = c / a.P;
    dst = reinterpret_cast<T*>(a.xh) + (long long)h * a.Pp + (c - h * a.P);
    step = (long long)a.H * a.Pp;
  } else {
    const bool is_b = c < n + gn;
    const int e = c - n - (is_b ? 0 : gn), g = e / a.N;
    dst = reinterpret_cast<T*>(is_b ? a.bc : a.cc) + (long long)g * a.Np + (e - g * a.N);
    step = (long long)a.G * a.Np;
  }
  dst += ((long long)b * a.n + t0) * step;
  for (int t = t0; t < t1; t += PF) {
    LlRaw4<T> nx[PF];
#pragma unroll
    for (int u = 0; u < PF; ++u)
      if (t + PF + u < t1) nx[u].load(src + (t + PF + u) * a.ld_proj);
#pragma unroll
    for (int u = 0; u < PF; ++u) {
      if (t + u < t1) {
        float cur[4];
        in[u].expand(cur);
        float4 o;
        float* op = reinterpret_cast<float*>(&o);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float s = bias[e] + w[0][e] * cur[e];
#pragma unroll
          for (int k = 1; k < TAPS; ++k) s += w[k][e] * x[k - 1][e];
          op[e] = ll_silu_t<T>(s);
#pragma unroll
          for (int k = TAPS - 1; k > 0; --k) x[k][e] = x[k - 1][e];
          x[0][e] = cur[e];
        }
        ll_store4(dst, o);
        dst += step;
      }
      in[u] = nx[u];
    }
  }
  if (t0 == 0)                             // this block alone read the carried inputs of these channels
    for (int t = max(0, a.n - TAPS); t < a.n; ++t) {
      LlRaw4<T> r;
      r.load(src + t * a.ld_proj);
      r.store(ring + (long long)((p0 + t) % TAPS) * C);
    }
}

// ---------------------------------------------------------------------------------------------- recurrence
// Block = (32 head dimensions, head, sequence): 32 rows of the state x 8 lanes, a lane holds NR state values of its row
// (columns r4 * 32 + slice * 4 + k, so that the eight lanes of a row read 128 consecutive bytes).
template <int NR>
struct LlState {
  float s[NR];
  __device__ __forceinline__ void load(const float* row, int Ns, int slice, bool zero) {
#pragma unroll
    for (int r = 0; r < NR / 4; ++r) {
      const int c = r * 32 + slice * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!zero && c < Ns) v = *reinterpret_cast<const float4*>(row + c);
      s[4 * r] = v.x; s[4 * r + 1] = v.y; s[4 * r + 2] = v.z; s[4 * r + 3] = v.w;
    }
  }
  __device__ __forceinline__ void store(float* row, int Ns, int slice) const {
#pragma unroll
    for (int r = 0; r < NR / 4; ++r) {
      const int c = r * 32 + slice * 4;
      if (c < Ns) *reinterpret_cast<float4*>(row + c) = make_float4(s[4 * r], s[4 * r + 1], s[4 * r + 2], s[4 * r + 3]);
    }
  }
  // S <- decay * S + (dt * x) B^T; returns this lane's part of S C
  __device__ __forceinline__ float step(float decay, float dtx, const float* B, const float* C, int slice) {
    float y = 0.f;
#pragma unroll
    for (int r = 0; r < NR / 4; ++r) {
      const float4 b = *reinterpret_cast<const float4*>(B + r * 32 + slice * 4);
      const float4 c = *reinterpret_cast<const float4*>(C + r * 32 + slice * 4);
      s[4 * r] = s[4 * r] * decay + dtx * b.x;             y += s[4 * r] * c.x;
      s[4 * r + 1] = s[4 * r + 1] * decay + dtx * b.y;     y += s[4 * r + 1] * c.y;
      s[4 * r + 2] = s[4 * r + 2] * decay + dtx * b.z;     y += s[4 * r + 2] * c.z;
      s[4 * r + 3] = s[4 * r + 3] * decay + dtx * b.w;     y += s[4 * r + 3] * c.w;
    }
    return y;
  }
};

__device__ __forceinline__ float ll_sum8(float v) {
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  return v;
}

template <typename T, int NR>
__global__ void __launch_bounds__(256) ll_scan_kernel(const __grid_constant__ gb_ll_mamba_args a) {
  pdl_wait();
  constexpr int TT = 16, NW = NR * 8;
  __shared__ __align__(16) float sB[TT][NW], sC[TT][NW];
  __shared__ float sX[TT][32], sDt[TT], sA[TT], sY[TT][33];
  const int h = blockIdx.y, b = blockIdx.z, pt = blockIdx.x * 32, g = h / (a.H / a.G);
  const int tid = threadIdx.x, pr = tid >> 3, slice = tid & 7, p = pt + pr;
  const int n = a.H * a.P, dt_col = 2 * n + 2 * a.G * a.N + h;
  const bool live = p < a.P;
  float* srow = a.ssm + (((long long)b * a.H + h) * a.P + (live ? p : 0)) * a.Ns;
  LlState<NR> S;
  S.load(srow, a.Ns, slice, a.st[b].abs_pos == 0 || !live);
  const float na = -expf(a.A_log[h]), bias = a.dt_bias[h], D = a.D[h];
  for (int t0 = 0; t0 < a.n; t0 += TT) {
    const int tn = min(TT, a.n - t0);
    const long long r0 = (long long)b * a.n + t0;
    __syncthreads();
    for (int i = tid; i < TT * NW; i += 256) {
      const int t = i / NW, c = i - t * NW;
      const bool ok = t < tn && c < a.N;
      const long long at = ((r0 + t) * a.G + g) * a.Np + c;
      sB[t][c] = ok ? Cvt<T>::to_f(reinterpret_cast<const T*>(a.bc)[at]) : 0.f;
      sC[t][c] = ok ? Cvt<T>::to_f(reinterpret_cast<const T*>(a.cc)[at]) : 0.f;
    }
    for (int i = tid; i < TT * 32; i += 256) {
      const int t = i >> 5, c = i & 31;
      sX[t][c] = (t < tn && pt + c < a.P) ? Cvt<T>::to_f(reinterpret_cast<const T*>(a.xh)[((r0 + t) * a.H + h) * a.Pp + pt + c]) : 0.f;
    }
    if (tid < tn) {
      const float dt = ll_softplus(Cvt<T>::to_f(reinterpret_cast<const T*>(a.proj)[(r0 + tid) * a.ld_proj + dt_col]) + bias);
      sDt[tid] = dt;
      sA[tid] = expf(na * dt);
    }
    __syncthreads();
    for (int t = 0; t < tn; ++t) {
      const float x = sX[t][pr];
      const float y = ll_sum8(S.step(sA[t], sDt[t] * x, sB[t], sC[t], slice));
      if (slice == 0) sY[t][pr] = y + D * x;
    }
    __syncthreads();
    for (int i = tid; i < tn * 32; i += 256) {
      const int t = i >> 5, c = i & 31;
      if (pt + c < a.P) reinterpret_cast<T*>(a.y)[(r0 + t) * a.ld_y + h * a.P + pt + c] = Cvt<T>::from_f(sY[t][c]);
    }
  }
  if (live) S.store(srow, a.Ns, slice);
}

// One token: convolution of this head's channels and of its group's B and C, then the recurrence.  The carried inputs
// are a ring of `taps` rows, so the new row never overwrites one that another block still reads.
template <typename T, int NR>
__global__ void __launch_bounds__(256) ll_mamba_step_kernel(const __grid_constant__ gb_ll_mamba_args a) {
  pdl_wait();
  constexpr int NW = NR * 8;
  __shared__ __align__(16) float sB[NW], sC[NW];
  __shared__ float sX[32];
  const int h = blockIdx.y, b = blockIdx.z, pt = blockIdx.x * 32, rep = a.H / a.G, g = h / rep;
  const int tid = threadIdx.x, pr = tid >> 3, slice = tid & 7, p = pt + pr;
  const int n = a.H * a.P, gn = a.G * a.N, C = n + 2 * gn, pos = a.st[b].abs_pos;
  const T* row = reinterpret_cast<const T*>(a.proj) + b * a.ld_proj;
  T* ring = reinterpret_cast<T*>(a.conv_state) + (long long)b * a.taps * C;
  const bool live = p < a.P;
  float* srow = a.ssm + (((long long)b * a.H + h) * a.P + (live ? p : 0)) * a.Ns;
  LlState<NR> S;
  S.load(srow, a.Ns, slice, pos == 0 || !live);
  const bool owner = (h % rep) == 0 && blockIdx.x == 0;      // writes the group's B and C inputs
  for (int i = tid; i < 32 + 2 * NW; i += 256) {
    int c = -1;
    if (i < 32) { if (pt + i < a.P) c = h * a.P + pt + i; }
    else {
      const int e = (i - 32) % NW, which = (i - 32) / NW;
      if (e < a.N) c = n + which * gn + g * a.N + e;
    }
    float v = 0.f;
    if (c >= 0) {
      const T cur = row[n + c];
      float s = a.conv_b[c] + a.conv_w[(long long)c * a.taps + a.taps - 1] * Cvt<T>::to_f(cur);
      for (int k = 1; k < a.taps; ++k)
        if (pos - k >= 0) s += a.conv_w[(long long)c * a.taps + a.taps - 1 - k] * Cvt<T>::to_f(ring[(long long)((pos - k) % a.taps) * C + c]);
      v = Cvt<T>::to_f(Cvt<T>::from_f(ll_silu_t<T>(s)));
      if (i < 32 || owner) ring[(long long)(pos % a.taps) * C + c] = cur;
    }
    if (i < 32) sX[i] = v;
    else if (i < 32 + NW) sB[i - 32] = v;
    else sC[i - 32 - NW] = v;
  }
  const float dt = ll_softplus(Cvt<T>::to_f(row[2 * n + 2 * gn + h]) + a.dt_bias[h]);
  const float decay = expf(-expf(a.A_log[h]) * dt);
  __syncthreads();
  const float x = sX[pr];
  const float y = ll_sum8(S.step(decay, dt * x, sB, sC, slice)) + a.D[h] * x;
  if (live) S.store(srow, a.Ns, slice);
  if (a.gated == nullptr) {
    if (live && slice == 0) reinterpret_cast<T*>(a.y)[b * a.ld_y + h * a.P + p] = Cvt<T>::from_f(y);
    return;
  }
  // y silu(z) for the norm that follows, and this block's part of its sum of squares
  __shared__ float s_sq[8];
  float v = 0.f;
  if (live && slice == 0) {
    v = Cvt<T>::to_f(Cvt<T>::from_f(y)) * ll_silu_t<T>(Cvt<T>::to_f(row[h * a.P + p]));
    a.gated[(long long)b * n + h * a.P + p] = v;
  }
  v = warp_sum(v * v);
  if ((tid & 31) == 0) s_sq[tid >> 5] = v;
  __syncthreads();
  if (tid == 0) {
    float q = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) q += s_sq[w];
    a.gated_sq[((long long)b * a.H + h) * gridDim.x + blockIdx.x] = q;
  }
}

// ---------------------------------------------------------------------------------------------- gated group norm
// One block of 128 threads per (row, part).
template <typename T>
__global__ void __launch_bounds__(128) ll_gated_norm_kernel(const __grid_constant__ gb_ll_mamba_args a) {
  pdl_wait();
  __shared__ float red[4];
  const int n = a.H * a.P, per = n / a.norm_groups, tid = threadIdx.x;
  const long long r = blockIdx.x;
  const int c0 = blockIdx.y * per;
  const T* y = reinterpret_cast<const T*>(a.y) + r * a.ld_y + c0;
  const T* z = reinterpret_cast<const T*>(a.proj) + r * a.ld_proj + c0;
  T* o = reinterpret_cast<T*>(a.out) + r * a.ld_out + c0;
  constexpr int KEEP = 16;
  float v[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = tid + 128 * k;
    v[k] = i < per ? Cvt<T>::to_f(y[i]) * ll_silu_t<T>(Cvt<T>::to_f(z[i])) : 0.f;
    ss += v[k] * v[k];
  }
  for (int i = tid + 128 * KEEP; i < per; i += 128) {
    const float u = Cvt<T>::to_f(y[i]) * ll_silu_t<T>(Cvt<T>::to_f(z[i]));
    ss += u * u;
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  const float inv = ll_inv_rms(red[0] + red[1] + red[2] + red[3], per, a.eps);
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = tid + 128 * k;
    if (i < per) o[i] = Cvt<T>::from_f(v[k] * inv * a.norm_w[c0 + i]);
  }
  for (int i = tid + 128 * KEEP; i < per; i += 128)
    o[i] = Cvt<T>::from_f(Cvt<T>::to_f(y[i]) * ll_silu_t<T>(Cvt<T>::to_f(z[i])) * inv * a.norm_w[c0 + i]);
}

// The same with 16-byte accesses: VPT vectors of eight values per thread.
template <typename T, int VPT>
__global__ void __launch_bounds__(256) ll_gated_norm_vec_kernel(const __grid_constant__ gb_ll_mamba_args a) {
  pdl_wait();
  __shared__ float red[8];
  const int per = a.H * a.P / a.norm_groups, tid = threadIdx.x, nv = per >> 3;
  const long long r = blockIdx.x;
  const int c0 = blockIdx.y * per;
  const T* y = reinterpret_cast<const T*>(a.y) + r * a.ld_y + c0;
  const T* z = reinterpret_cast<const T*>(a.proj) + r * a.ld_proj + c0;
  T* o = reinterpret_cast<T*>(a.out) + r * a.ld_out + c0;
  float v[VPT][8], zz[VPT][8];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = tid + blockDim.x * k;
    if (i < nv) { ll_load8(y + 8 * i, v[k]); ll_load8(z + 8 * i, zz[k]); }
  }
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    if (tid + blockDim.x * k >= nv) break;
#pragma unroll
    for (int e = 0; e < 8; ++e) { v[k][e] *= ll_silu_t<T>(zz[k][e]); ss += v[k][e] * v[k][e]; }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) tot += red[w];
  const float inv = ll_inv_rms(tot, per, a.eps);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = tid + blockDim.x * k;
    if (i >= nv) break;
    float g[8];
    ll_load8(a.norm_w + c0 + 8 * i, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[k][e] *= inv * g[e];
    ll_store8(o + 8 * i, v[k]);
  }
}

static bool ll_vec_ok(const gb_ll_mamba_args& a) {
  return a.P % 8 == 0 && a.N % 8 == 0 && a.Pp % 8 == 0 && a.Np % 8 == 0 && a.ld_proj % 8 == 0 && a.ld_y % 8 == 0 && a.ld_out % 8 == 0 &&
         ((reinterpret_cast<uintptr_t>(a.proj) | reinterpret_cast<uintptr_t>(a.xh) | reinterpret_cast<uintptr_t>(a.bc) |
           reinterpret_cast<uintptr_t>(a.cc) | reinterpret_cast<uintptr_t>(a.conv_state) | reinterpret_cast<uintptr_t>(a.y) |
           reinterpret_cast<uintptr_t>(a.out) | reinterpret_cast<uintptr_t>(a.norm_w) | reinterpret_cast<uintptr_t>(a.conv_w) |
           reinterpret_cast<uintptr_t>(a.conv_b)) & 15) == 0;
}

template <typename T>
static int ll_scan_go(const gb_ll_mamba_args& a, bool step, cudaStream_t st) {
  const dim3 grid((a.P + 31) / 32, a.H, a.B);
#define GO(NR) do { if (step) GB_PDL_LAUNCH((ll_mamba_step_kernel<T, NR>), grid, dim3(256), st, a); \
                    else GB_PDL_LAUNCH((ll_scan_kernel<T, NR>), grid, dim3(256), st, a); } while (0)
  if (a.N <= 64) GO(8);
  else if (a.N <= 128) GO(16);
  else GO(32);
#undef GO
  return gb_launch_rc();
}

template <typename T>
static int ll_conv_go(const gb_ll_mamba_args& a, cudaStream_t st) {
  const int C = a.H * a.P + 2 * a.G * a.N;
  // tokens per thread: long enough to pay for loading the taps, short enough to fill the machine
  const long long groups = (long long)((C / 4 + 127) / 128) * a.B;
  int tile = 64;
  while (tile > 8 && groups * ((a.n + tile - 1) / tile) < 148 * 6) tile >>= 1;
  if (ll_vec_ok(a) && a.taps >= 2 && a.taps <= 4 && (a.n + tile - 1) / tile <= 65535) {
    const dim3 vg((C / 4 + 127) / 128, (a.n + tile - 1) / tile, a.B);
    if (a.taps == 2) GB_PDL_LAUNCH((ll_conv_vec_kernel<T, 2>), vg, dim3(128), st, a, tile);
    else if (a.taps == 3) GB_PDL_LAUNCH((ll_conv_vec_kernel<T, 3>), vg, dim3(128), st, a, tile);
    else GB_PDL_LAUNCH((ll_conv_vec_kernel<T, 4>), vg, dim3(128), st, a, tile);
    return gb_launch_rc();
  }
  const dim3 grid((C + 127) / 128, (a.n + CONV_TT - 1) / CONV_TT, a.B);
  if (a.taps <= 4) GB_PDL_LAUNCH((ll_conv_kernel<T, 4>), grid, dim3(128), st, a);
  else if (a.taps <= 8) GB_PDL_LAUNCH((ll_conv_kernel<T, 8>), grid, dim3(128), st, a);
  else GB_PDL_LAUNCH((ll_conv_kernel<T, 32>), grid, dim3(128), st, a);
  return gb_launch_rc();
}

}  // namespace gb

using namespace gb;

static int ll_mamba_check(const gb_ll_mamba_args* p) {
  if (!p || !p->st || !p->proj || p->B <= 0 || p->n <= 0 || p->H <= 0 || p->G <= 0 || p->H % p->G || p->P <= 0 || p->N <= 0) return -1;
  if (p->taps < 1 || p->taps > 32 || p->N > 256 || p->Pp < p->P || p->Np < p->N || p->Ns < p->N || p->Ns % 4) return -2;
  if (!p->conv_w || !p->conv_b || !p->dt_bias || !p->A_log || !p->D || !p->conv_state || !p->ssm || !p->y) return -1;
  return p->dtype == 1 || p->dtype == 2 ? 0 : -6;
}

extern "C" int gb_ll_conv(const gb_ll_mamba_args* p, cudaStream_t st) {
  if (const int rc = ll_mamba_check(p)) return rc;
  if (!p->xh || !p->bc || !p->cc) return -1;
  return p->dtype == 1 ? ll_conv_go<__nv_bfloat16>(*p, st) : ll_conv_go<float>(*p, st);
}

extern "C" int gb_ll_scan(const gb_ll_mamba_args* p, cudaStream_t st) {
  if (const int rc = ll_mamba_check(p)) return rc;
  if (!p->xh || !p->bc || !p->cc) return -1;
  return p->dtype == 1 ? ll_scan_go<__nv_bfloat16>(*p, false, st) : ll_scan_go<float>(*p, false, st);
}

extern "C" int gb_ll_mamba_step(const gb_ll_mamba_args* p, cudaStream_t st) {
  if (const int rc = ll_mamba_check(p)) return rc;
  if (p->n != 1) return -3;
  if (p->gated && !p->gated_sq) return -1;
  return p->dtype == 1 ? ll_scan_go<__nv_bfloat16>(*p, true, st) : ll_scan_go<float>(*p, true, st);
}

extern "C" int gb_ll_gated_norm(const gb_ll_mamba_args* p, cudaStream_t st) {
  if (const int rc = ll_mamba_check(p)) return rc;
  if (!p->out || !p->norm_w || p->norm_groups <= 0 || (p->H * p->P) % p->norm_groups) return -1;
  const dim3 grid(p->B * p->n, p->norm_groups);
  const int per = p->H * p->P / p->norm_groups;
  if (per % 8 == 0 && per <= 8192 && ll_vec_ok(*p)) {
    const int nv = per / 8, threads = nv >= 256 ? 256 : (nv + 31) / 32 * 32, vpt = (nv + threads - 1) / threads;
#define GN(T, V) GB_PDL_LAUNCH((ll_gated_norm_vec_kernel<T, V>), grid, dim3(threads), st, *p)
#define GNT(T) do { if (vpt == 1) GN(T, 1); else if (vpt == 2) GN(T, 2); else if (vpt == 3) GN(T, 3); else GN(T, 4); } while (0)
    if (p->dtype == 1) GNT(__nv_bfloat16);
    else GNT(float);
#undef GNT
#undef GN
    return gb_launch_rc();
  }
  if (p->dtype == 1) GB_PDL_LAUNCH(ll_gated_norm_kernel<__nv_bfloat16>, grid, dim3(128), st, *p);
  else GB_PDL_LAUNCH(ll_gated_norm_kernel<float>, grid, dim3(128), st, *p);
  return gb_launch_rc();
}
