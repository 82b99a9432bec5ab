// Attention of layer-list models on CUDA cores (interface in gb_layers.h): what every head size and fp32 run on, and the
// token step.  Keys live in one cache per layer: the first `keep` positions stay, later positions share a ring.  The keys
// a query range can see are enumerated as one list (kept positions, then the window), so no slot outside it is read.
#include <type_traits>

#include "sm100_common.cuh"
#include "gb_layers.h"
#include "layers_util.cuh"

namespace gb {

// Angle of a pair at a position: the product in double, reduced to one turn, then an fp32 cosine and sine.
__device__ __forceinline__ float2 ll_rotation(int pos, double freq) {
  double ang = (double)pos * freq;
  ang -= 6.283185307179586476925 * rint(ang * 0.159154943091895335769);
  float sn, cs;
  sincosf((float)ang, &sn, &cs);
  return make_float2(cs, sn);
}

__device__ __forceinline__ float ll_query_temperature(int pos, float coef, int every) {
  return 1.f + coef * logf((float)((pos + 1) / every + 1));
}

// Score as the soft-max sees it: scaled, capped, less the slope times the distance.
// (T of 16 bits: tanh(z) = 1 - 2 / (e^2z + 1) with the hardware's exponential and quotient, about 1e-6 of the cap.)
template <typename T>
__device__ __forceinline__ float ll_score(float dot, float scale, float cap, float slope, int back) {
  float s = dot * scale;
  if (cap > 0.f) s = sizeof(T) == 4 ? cap * tanhf(s / cap) : cap - __fdividef(2.f * cap, 1.f + __expf(fminf(__fdividef(2.f * s, cap), 80.f)));
  return s - slope * (float)back;
}

__global__ void __launch_bounds__(256) ll_rotations_kernel(const double* __restrict__ freq, int pairs, const gb_seq_state* __restrict__ st,
                                                           int n, long long total, float2* __restrict__ cs) {
  pdl_wait();
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= total) return;
  const int r = (int)(i / pairs), b = r / n;
  cs[i] = ll_rotation(st[b].abs_pos + r - b * n, freq[i - (long long)r * pairs]);
}

// LPH lanes per head, eight dimensions per lane (head sizes and offsets in multiples of eight, interleaved pairs).
template <typename T, int LPH>
__global__ void __launch_bounds__(256) ll_qkv_store_vec_kernel(const __grid_constant__ gb_ll_attn_args a) {
  pdl_wait();
  const int heads = a.H + 2 * a.G;
  const int lane = threadIdx.x & 31, sub = lane % LPH, c = sub * 8;
  const long long item = (blockIdx.x * 8LL + (threadIdx.x >> 5)) * (32 / LPH) + lane / LPH;
  const bool live = item < (long long)a.B * a.n * heads;
  const int r = live ? (int)(item / heads) : 0, h = live ? (int)(item - (long long)r * heads) : 0;
  const int b = r / a.n, pos = a.st[b].abs_pos + r - b * a.n;
  const T* row = reinterpret_cast<const T*>(a.proj) + r * a.ld_proj;
  const long long crow = (long long)b * a.cap + ll_ring_row(pos, a.keep, a.cap);
  const bool is_v = h >= a.H + a.G;
  const int d = is_v ? a.dv : a.dk, dp = is_v ? a.dvp : a.dkp;
  const T* src = is_v ? row + (a.H + a.G) * a.dk + (h - a.H - a.G) * a.dv : row + h * a.dk;
  T* dst = is_v ? reinterpret_cast<T*>(a.cache_v) + (crow * a.G + (h - a.H - a.G)) * a.dvp
                : h < a.H ? reinterpret_cast<T*>(a.q) + ((long long)r * a.H + h) * a.dkp
                          : reinterpret_cast<T*>(a.cache_k) + (crow * a.G + (h - a.H)) * a.dkp;
  float v[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] = 0.f;
  if (live && c < d) ll_load8(src + c, v);
  float ss = 0.f;
  if (!is_v) {
    if (c < a.rot_dims) {
      const float4* cs = reinterpret_cast<const float4*>(a.cs + (long long)r * a.rot_dims + c);
      const float4 p0 = cs[0], p1 = cs[1];
      const float cc[4] = {p0.x, p0.z, p1.x, p1.z}, sn[4] = {p0.y, p0.w, p1.y, p1.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float x = v[2 * e], y = v[2 * e + 1];
        v[2 * e] = x * cc[e] - y * sn[e];
        v[2 * e + 1] = y * cc[e] + x * sn[e];
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += v[e] * v[e];
  }
#pragma unroll
  for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!is_v && a.qk_norm) {
    const float inv = ll_inv_rms(ss, a.dk, a.eps);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= inv;
  }
  if (h < a.H && a.temp_every > 0) {
    const float f = ll_query_temperature(pos, a.temp_coef, a.temp_every);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= f;
  }
  if (live && c < dp) ll_store8(dst + c, v);
}

// One warp per (row, head) over the query, key and value heads of the fused projection.
template <typename T>
__global__ void __launch_bounds__(256) ll_qkv_store_kernel(const __grid_constant__ gb_ll_attn_args a) {
  pdl_wait();
  const int heads = a.H + 2 * a.G;
  const long long gw = blockIdx.x * 8LL + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (gw >= (long long)a.B * a.n * heads) return;
  const int r = (int)(gw / heads), h = (int)(gw - (long long)r * heads);
  const int b = r / a.n, t = r - b * a.n;
  const int pos = a.st[b].abs_pos + t;
  const T* row = reinterpret_cast<const T*>(a.proj) + r * a.ld_proj;
  const long long crow = (long long)b * a.cap + ll_ring_row(pos, a.keep, a.cap);
  if (h >= a.H + a.G) {
    const int g = h - a.H - a.G;
    const T* src = row + (a.H + a.G) * a.dk + g * a.dv;
    T* dst = reinterpret_cast<T*>(a.cache_v) + (crow * a.G + g) * a.dvp;
    for (int i = lane; i < a.dvp; i += 32) dst[i] = i < a.dv ? src[i] : Cvt<T>::from_f(0.f);
    return;
  }
  const T* src = row + h * a.dk;
  T* dst = h < a.H ? reinterpret_cast<T*>(a.q) + ((long long)r * a.H + h) * a.dkp
                   : reinterpret_cast<T*>(a.cache_k) + (crow * a.G + (h - a.H)) * a.dkp;
  // lane l holds dimensions l, l + 32, ...; the partner of a rotated dimension comes from memory again (same cache line)
  const int half = a.rot_dims / 2;
  float v[8];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < 8; ++k) {
    const int i = lane + 32 * k;
    v[k] = 0.f;
    if (i < a.dk) {
      float x = Cvt<T>::to_f(src[i]);
      if (i < a.rot_dims) {
        const int pair = a.rot_half ? (i < half ? i : i - half) : i >> 1;
        const bool second = a.rot_half ? i >= half : (i & 1);
        const int pi = a.rot_half ? (second ? i - half : i + half) : i ^ 1;
        const float xp = Cvt<T>::to_f(src[pi]);
        const float2 cs = a.cs ? reinterpret_cast<const float2*>(a.cs)[(long long)r * half + pair] : ll_rotation(pos, a.freq[pair]);
        x = second ? x * cs.x + xp * cs.y : x * cs.x - xp * cs.y;
      }
      v[k] = x;
      ss += x * x;
    }
  }
  float inv = 1.f;
  if (a.qk_norm) inv = ll_inv_rms(warp_sum(ss), a.dk, a.eps);
  if (h < a.H && a.temp_every > 0) inv *= ll_query_temperature(pos, a.temp_coef, a.temp_every);
#pragma unroll
  for (int k = 0; k < 8; ++k) {
    const int i = lane + 32 * k;
    if (i < a.dkp) dst[i] = Cvt<T>::from_f(i < a.dk ? v[k] * inv : 0.f);
  }
}

template <int N>
__device__ __forceinline__ float ll_group_sum(float v) {
#pragma unroll
  for (int o = N / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Range of keys for queries at positions [p_first, p_last]: kept [0, n_kept), then positions [win_lo, p_last].
struct LlKeyRange { int n_kept, win_lo, count; };
__device__ __forceinline__ LlKeyRange ll_key_range(int p_first, int p_last, int window, int keep) {
  LlKeyRange k;
  k.n_kept = min(keep, p_last + 1);
  k.win_lo = max(keep, window > 0 ? p_first - window + 1 : 0);
  k.count = k.n_kept + max(0, p_last - k.win_lo + 1);
  return k;
}

// HD / 16 threads per query row, each with 16 of the head's dimensions; key tiles of 32 in shared memory as fp32.
template <typename T, int HD>
__global__ void __launch_bounds__(128) ll_attn_prefill_kernel(const __grid_constant__ gb_ll_attn_args a) {
  pdl_wait();
  constexpr int TPR = HD / 16, ROWS = 128 / TPR, KT = 32;
  extern __shared__ __align__(16) float la_dyn[];
  float* sK = la_dyn;
  float* sV = sK + KT * a.dkp;
  int* sPos = reinterpret_cast<int*>(sV + KT * a.dvp);
  const int b = blockIdx.z, h = blockIdx.y, q0 = blockIdx.x * ROWS, g = h / (a.H / a.G);
  const int r = threadIdx.x / TPR, sub = threadIdx.x % TPR;
  const int t = q0 + r, p0 = a.st[b].abs_pos, i = p0 + t;
  const bool live = t < a.n;
  const long long row = (long long)b * a.n + t;
  float q[16], o[16];
#pragma unroll
  for (int d = 0; d < 16; ++d) {
    const int c = sub * 16 + d;
    q[d] = (live && c < a.dkp) ? Cvt<T>::to_f(reinterpret_cast<const T*>(a.q)[(row * a.H + h) * a.dkp + c]) : 0.f;
    o[d] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const float slope = a.slopes ? a.slopes[h] : 0.f;
  const LlKeyRange kr = ll_key_range(p0 + q0, p0 + min(a.n, q0 + ROWS) - 1, a.window, a.keep);
  for (int e0 = 0; e0 < kr.count; e0 += KT) {
    __syncthreads();
    for (int x = threadIdx.x; x < KT; x += 128) {
      const int e = e0 + x;
      sPos[x] = e < kr.n_kept ? e : e < kr.count ? kr.win_lo + (e - kr.n_kept) : -1;
    }
    __syncthreads();
    for (int x = threadIdx.x; x < KT * a.dkp; x += 128) {
      const int kk = x / a.dkp, c = x - kk * a.dkp, p = sPos[kk];
      sK[x] = p < 0 ? 0.f : Cvt<T>::to_f(reinterpret_cast<const T*>(a.cache_k)[((long long)b * a.cap + ll_ring_row(p, a.keep, a.cap)) * a.ld_k + g * a.dkp + c]);
    }
    for (int x = threadIdx.x; x < KT * a.dvp; x += 128) {
      const int kk = x / a.dvp, c = x - kk * a.dvp, p = sPos[kk];
      sV[x] = p < 0 ? 0.f : Cvt<T>::to_f(reinterpret_cast<const T*>(a.cache_v)[((long long)b * a.cap + ll_ring_row(p, a.keep, a.cap)) * a.ld_v + g * a.dvp + c]);
    }
    __syncthreads();
    const int kn = min(KT, kr.count - e0);
    for (int kk = 0; kk < kn; ++kk) {
      const int p = sPos[kk];
      float s = 0.f;
#pragma unroll
      for (int d = 0; d < 16; ++d) {
        const int c = sub * 16 + d;
        if (c < a.dkp) s += q[d] * sK[kk * a.dkp + c];
      }
      s = ll_score<T>(ll_group_sum<TPR>(s), a.scale, a.softcap, slope, i - p);
      if (!live || p > i || !(a.window <= 0 || i - p < a.window || p < a.keep)) continue;
      const float mn = fmaxf(m, s);
      const float corr = expf(m - mn), pr = expf(s - mn);
      l = l * corr + pr;
#pragma unroll
      for (int d = 0; d < 16; ++d) {
        const int c = sub * 16 + d;
        o[d] = o[d] * corr + (c < a.dvp ? pr * sV[kk * a.dvp + c] : 0.f);
      }
      m = mn;
    }
  }
  if (!live) return;
  float fac = 1.f;
  if (a.sink) {
    const float sk = a.sink[h], mn = fmaxf(m, sk);
    fac = expf(m - mn);
    l = l * fac + expf(sk - mn);
  }
  fac = l > 0.f ? fac / l : 0.f;
  const T* gate = reinterpret_cast<const T*>(a.gate) + row * a.ld_gate + h * a.dv;
  T* op = reinterpret_cast<T*>(a.out) + row * a.ldo + h * a.dv;
#pragma unroll
  for (int d = 0; d < 16; ++d) {
    const int c = sub * 16 + d;
    if (c < a.dv) {
      float v = o[d] * fac;
      if (a.gate) v *= ll_sigmoid(Cvt<T>::to_f(gate[c]));
      op[c] = Cvt<T>::from_f(v);
    }
  }
}

// ---------------------------------------------------------------------------------------------- token step
// grid (B * G * ceil(R / GQ), splits), 4 warps; R = H / G query heads share a key/value head, GQ of them per block.  A lane
// holds EPL consecutive dimensions; each warp walks its keys with an online soft-max per query head.
template <typename T, int EPL>
__device__ __forceinline__ void ll_load(const T* p, float (&v)[EPL]) {
  if constexpr (std::is_same<T, float>::value) {
#pragma unroll
    for (int e = 0; e < EPL; e += 2) { const float2 f = *reinterpret_cast<const float2*>(p + e); v[e] = f.x; v[e + 1] = f.y; }
  } else {
#pragma unroll
    for (int e = 0; e < EPL; e += 2) { const float2 f = Cvt<T>::unpack2(*reinterpret_cast<const uint32_t*>(p + e)); v[e] = f.x; v[e + 1] = f.y; }
  }
}

template <typename T, int EPL, int GQ>
__global__ void __launch_bounds__(128) ll_attn_decode_kernel(const __grid_constant__ gb_ll_attn_args a) {
  pdl_wait();
  constexpr int HD = EPL * 32;
  const int R = a.H / a.G, chunks = (R + GQ - 1) / GQ;
  const int b = blockIdx.x / (a.G * chunks), rem = blockIdx.x - b * a.G * chunks;
  const int g = rem / chunks, h0 = g * R + (rem - g * chunks) * GQ, nh = min(GQ, (g + 1) * R - h0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, split = blockIdx.y;
  const int pos = a.st[b].abs_pos;
  const LlKeyRange kr = ll_key_range(pos, pos, a.window, a.keep);
  const int per = (kr.count + a.splits - 1) / a.splits;
  const int lo = split * per, hi = min(kr.count, lo + per);
  const bool kl = lane * EPL < a.dkp, vl = lane * EPL < a.dvp;
  float q[GQ][EPL], o[GQ][EPL], m[GQ], l[GQ], slope[GQ];
#pragma unroll
  for (int x = 0; x < GQ; ++x) {
    m[x] = -INFINITY; l[x] = 0.f;
    slope[x] = a.slopes && x < nh ? a.slopes[h0 + x] : 0.f;
#pragma unroll
    for (int e = 0; e < EPL; ++e) { q[x][e] = 0.f; o[x][e] = 0.f; }
    if (x < nh && kl) ll_load<T, EPL>(reinterpret_cast<const T*>(a.q) + ((long long)b * a.H + h0 + x) * a.dkp + lane * EPL, q[x]);
  }
  constexpr int KB = EPL <= 4 ? 4 : 2;            // keys in flight per warp: all their loads come before the first use
  for (int e0 = lo + warp * KB; e0 < hi; e0 += 4 * KB) {
    float kf[KB][EPL], vf[KB][EPL];
    int back[KB];
#pragma unroll
    for (int j = 0; j < KB; ++j) {
      const int e = min(e0 + j, hi - 1);
      const int p = e < kr.n_kept ? e : kr.win_lo + (e - kr.n_kept);
      back[j] = pos - p;
      const long long crow = (long long)b * a.cap + ll_ring_row(p, a.keep, a.cap);
#pragma unroll
      for (int x = 0; x < EPL; ++x) { kf[j][x] = 0.f; vf[j][x] = 0.f; }
      if (kl) ll_load<T, EPL>(reinterpret_cast<const T*>(a.cache_k) + crow * a.ld_k + g * a.dkp + lane * EPL, kf[j]);
      if (vl) ll_load<T, EPL>(reinterpret_cast<const T*>(a.cache_v) + crow * a.ld_v + g * a.dvp + lane * EPL, vf[j]);
    }
#pragma unroll
    for (int x = 0; x < GQ; ++x) {
      float s[KB], mn = m[x];
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        s[j] = 0.f;
#pragma unroll
        for (int e = 0; e < EPL; ++e) s[j] += q[x][e] * kf[j][e];
      }
#pragma unroll
      for (int d = 16; d > 0; d >>= 1)
#pragma unroll
        for (int j = 0; j < KB; ++j) s[j] += __shfl_xor_sync(0xffffffffu, s[j], d);
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        s[j] = e0 + j < hi ? ll_score<T>(s[j], a.scale, a.softcap, slope[x], back[j]) : -INFINITY;
        mn = fmaxf(mn, s[j]);
      }
      const float c = expf(m[x] - mn);            // the first key of a group is always real, so mn is finite
      l[x] *= c;
#pragma unroll
      for (int e = 0; e < EPL; ++e) o[x][e] *= c;
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        const float pr = expf(s[j] - mn);
        l[x] += pr;
#pragma unroll
        for (int e = 0; e < EPL; ++e) o[x][e] += pr * vf[j][e];
      }
      m[x] = mn;
    }
  }
  __shared__ float sm_m[4][GQ], sm_l[4][GQ], sm_o[4][GQ][HD];
#pragma unroll
  for (int x = 0; x < GQ; ++x) {
    if (lane == 0) { sm_m[warp][x] = m[x]; sm_l[warp][x] = l[x]; }
#pragma unroll
    for (int e = 0; e < EPL; ++e) sm_o[warp][x][lane * EPL + e] = o[x][e];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * a.dvp; i += 128) {
    const int x = i / a.dvp, c = i - x * a.dvp;
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, sm_m[w][x]);
    float ll = 0.f, oo = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = sm_m[w][x] == -INFINITY ? 0.f : expf(sm_m[w][x] - mm);
      ll += sm_l[w][x] * f;
      oo += sm_o[w][x][c] * f;
    }
    const long long at = ((long long)b * a.H + h0 + x) * a.splits + split;
    a.scratch[at * a.dvp + c] = oo;
    if (c == 0) *reinterpret_cast<float2*>(a.scratch + (long long)a.B * a.H * a.splits * a.dvp + 2 * at) = make_float2(mm, ll);
  }
}

// One block per (sequence, head): the splits' results, the sink and the output gate.  Groups of threads take every g-th split.
template <typename T>
__global__ void __launch_bounds__(256) ll_attn_merge_kernel(const __grid_constant__ gb_ll_attn_args a) {
  pdl_wait();
  __shared__ float s_f[128];
  __shared__ float s_red[8];
  __shared__ __align__(16) float s_p[256 * 4];
  const int b = blockIdx.x / a.H, h = blockIdx.x - b * a.H, tid = threadIdx.x;
  const int quads = a.dvp / 4, ng = min(a.splits, 256 / quads), g = tid / quads, q = tid - g * quads;
  const long long at = ((long long)b * a.H + h) * a.splits;
  const float* base = a.scratch + at * a.dvp + 4 * q;
  const float2* ml = reinterpret_cast<const float2*>(a.scratch + (long long)a.B * a.H * a.splits * a.dvp + 2 * at);
  constexpr int AHEAD = 4;
  float4 v[AHEAD];
#pragma unroll
  for (int k = 0; k < AHEAD; ++k)
    if (g < ng && g + k * ng < a.splits) v[k] = *reinterpret_cast<const float4*>(base + (long long)(g + k * ng) * a.dvp);
  const float2 own = tid < a.splits ? ml[tid] : make_float2(-INFINITY, 0.f);       // up to 128 splits: the first four warps
  float mm = warp_max(own.x);
  if ((tid & 31) == 0 && tid < 128) s_red[tid >> 5] = mm;
  __syncthreads();
  mm = fmaxf(fmaxf(s_red[0], s_red[1]), fmaxf(s_red[2], s_red[3]));
  if (a.sink) mm = fmaxf(mm, a.sink[h]);
  const float f = own.x == -INFINITY ? 0.f : expf(own.x - mm);
  const float lw = warp_sum(own.y * f);
  if (tid < 128) {
    s_f[tid] = f;
    if ((tid & 31) == 0) s_red[4 + (tid >> 5)] = lw;
  }
  __syncthreads();
  float l = s_red[4] + s_red[5] + s_red[6] + s_red[7];
  if (a.sink) l += expf(a.sink[h] - mm);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  if (g < ng) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    auto add = [&](int s, const float4& x) {
      const float w = s_f[s];
      o.x += x.x * w; o.y += x.y * w; o.z += x.z * w; o.w += x.w * w;
    };
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
      if (g + k * ng < a.splits) add(g + k * ng, v[k]);
#pragma unroll 4
    for (int s = g + AHEAD * ng; s < a.splits; s += ng) add(s, *reinterpret_cast<const float4*>(base + (long long)s * a.dvp));
    *reinterpret_cast<float4*>(&s_p[tid * 4]) = o;
  }
  __syncthreads();
  const T* gate = reinterpret_cast<const T*>(a.gate) + b * a.ld_gate + h * a.dv;
  T* op = reinterpret_cast<T*>(a.out) + b * a.ldo + h * a.dv;
  for (int c = tid; c < a.dv; c += 256) {
    float o = 0.f;
    for (int k = 0; k < ng; ++k) o += s_p[k * a.dvp + c];
    float v1 = o * inv;
    if (a.gate) v1 *= ll_sigmoid(Cvt<T>::to_f(gate[c]));
    op[c] = Cvt<T>::from_f(v1);
  }
}

template <typename T, int EPL>
static void ll_decode_go(const gb_ll_attn_args& a, cudaStream_t st) {
  const int R = a.H / a.G;
#define GO(GQ) GB_PDL_LAUNCH((ll_attn_decode_kernel<T, EPL, GQ>), dim3(a.B * a.G * ((R + GQ - 1) / GQ), a.splits), dim3(128), st, a)
  if (R == 1) GO(1);
  else if (R == 2) GO(2);
  else GO(4);
#undef GO
  GB_PDL_LAUNCH(ll_attn_merge_kernel<T>, dim3(a.B * a.H), dim3(256), st, a);
}

template <typename T>
static int ll_prefill_go(const gb_ll_attn_args& a, cudaStream_t st) {
  const int hd = a.dkp > a.dvp ? a.dkp : a.dvp;
  const size_t smem = (size_t)32 * (a.dkp + a.dvp) * 4 + 32 * 4;
#define GO(HD) GB_PDL_LAUNCH_SMEM((ll_attn_prefill_kernel<T, HD>), dim3((a.n + 2048 / HD - 1) / (2048 / HD), a.H, a.B), dim3(128), smem, st, a)
  if (hd <= 64) GO(64);
  else if (hd <= 128) GO(128);
  else GO(256);
#undef GO
  return gb_launch_rc();
}

}  // namespace gb

using namespace gb;

static int ll_attn_check(const gb_ll_attn_args* p) {
  if (!p || !p->st || !p->q || !p->cache_k || !p->cache_v || p->B <= 0 || p->n <= 0 || p->G <= 0 || p->H <= 0 || p->H % p->G) return -1;
  if (p->dk <= 0 || p->dv <= 0 || p->dk > p->dkp || p->dv > p->dvp || p->dkp > 256 || p->dvp > 256 || p->dkp % 8 || p->dvp % 8) return -2;
  if (p->rot_dims < 0 || p->rot_dims % 2 || p->rot_dims > p->dk || (p->rot_dims > 0 && !p->freq)) return -3;
  if (p->keep < 0 || p->cap <= p->keep || p->window < 0 || p->ld_k < p->G * p->dkp || p->ld_v < p->G * p->dvp || p->temp_every < 0) return -4;
  // the positions one call can see have to be in the ring together (window == 0: the caller bounds the length)
  if (p->window > 0 && p->pos0_max >= 0) {
    const long long last = (long long)p->pos0_max + p->n;
    const long long need = (long long)p->window - 1 + p->n;
    if (last - p->keep > p->cap - p->keep && need > p->cap - p->keep) return -5;
  }
  if (p->window == 0 && p->pos0_max >= 0 && p->pos0_max + p->n > p->cap) return -5;
  return p->dtype == 1 || p->dtype == 2 ? 0 : -6;
}

extern "C" int gb_ll_rotations(const double* freq, int pairs, const gb_seq_state* st, int B, int n, float* cs, cudaStream_t stream) {
  if (!freq || !st || !cs || pairs <= 0 || B <= 0 || n <= 0) return -1;
  const long long total = (long long)B * n * pairs;
  GB_PDL_LAUNCH(ll_rotations_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), stream, freq, pairs, st, n, total, reinterpret_cast<float2*>(cs));
  return gb_launch_rc();
}

extern "C" int gb_ll_qkv_store(const gb_ll_attn_args* p, cudaStream_t st) {
  if (const int rc = ll_attn_check(p)) return rc;
  if (!p->proj || p->ld_k != p->G * p->dkp || p->ld_v != p->G * p->dvp) return -4;
  const long long items = (long long)p->B * p->n * (p->H + 2 * p->G);
  const bool vec = p->dk % 8 == 0 && p->dv % 8 == 0 && p->rot_dims % 8 == 0 && !p->rot_half && (p->cs || p->rot_dims == 0) && p->ld_proj % 8 == 0 &&
                   ((reinterpret_cast<uintptr_t>(p->proj) | reinterpret_cast<uintptr_t>(p->q) | reinterpret_cast<uintptr_t>(p->cache_k) |
                     reinterpret_cast<uintptr_t>(p->cache_v) | reinterpret_cast<uintptr_t>(p->cs)) & 15) == 0;
  if (vec) {
    const int hd = p->dkp > p->dvp ? p->dkp : p->dvp, lph = hd <= 64 ? 8 : hd <= 128 ? 16 : 32;
    const dim3 vg((unsigned)((items + 8 * (32 / lph) - 1) / (8 * (32 / lph))));
#define QV(T, L) GB_PDL_LAUNCH((ll_qkv_store_vec_kernel<T, L>), vg, dim3(256), st, *p)
    if (p->dtype == 1) { if (lph == 8) QV(__nv_bfloat16, 8); else if (lph == 16) QV(__nv_bfloat16, 16); else QV(__nv_bfloat16, 32); }
    else { if (lph == 8) QV(float, 8); else if (lph == 16) QV(float, 16); else QV(float, 32); }
#undef QV
    return gb_launch_rc();
  }
  const dim3 grid((unsigned)((items + 7) / 8));
  if (p->dtype == 1) GB_PDL_LAUNCH(ll_qkv_store_kernel<__nv_bfloat16>, grid, dim3(256), st, *p);
  else GB_PDL_LAUNCH(ll_qkv_store_kernel<float>, grid, dim3(256), st, *p);
  return gb_launch_rc();
}

extern "C" int gb_ll_attn_prefill(const gb_ll_attn_args* p, cudaStream_t st) {
  if (const int rc = ll_attn_check(p)) return rc;
  if (!p->out) return -1;
  return p->dtype == 1 ? ll_prefill_go<__nv_bfloat16>(*p, st) : ll_prefill_go<float>(*p, st);
}

extern "C" int gb_ll_attn_decode(const gb_ll_attn_args* p, cudaStream_t st) {
  if (const int rc = ll_attn_check(p)) return rc;
  if (!p->out || !p->scratch || p->n != 1 || p->splits < 1 || p->splits > 128) return -1;
  const int hd = p->dkp > p->dvp ? p->dkp : p->dvp;
  if (p->dtype == 1) {
    if (hd <= 64) ll_decode_go<__nv_bfloat16, 2>(*p, st);
    else if (hd <= 128) ll_decode_go<__nv_bfloat16, 4>(*p, st);
    else ll_decode_go<__nv_bfloat16, 8>(*p, st);
  } else {
    if (hd <= 64) ll_decode_go<float, 2>(*p, st);
    else if (hd <= 128) ll_decode_go<float, 4>(*p, st);
    else ll_decode_go<float, 8>(*p, st);
  }
  return gb_launch_rc();
}
