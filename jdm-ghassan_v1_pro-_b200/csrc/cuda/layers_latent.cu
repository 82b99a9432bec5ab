// Attention over a shared latent (interface in gb_layers.h): what it stores per position, and the path of a few new tokens, in
// which queries are taken through their head's key map so that all heads attend to the stored rows themselves.  A stored
// row is read once for a group of heads and serves as key and as value.
#include "sm100_common.cuh"
#include "gb_layers.h"
#include "layers_util.cuh"

namespace gb {

// Element e of a vector whose leading rot_dims turn in neighbouring pairs; cs: this row's cosines and sines.
template <typename T>
__device__ __forceinline__ float ll_turned(const T* src, int e, int rot_dims, const float2* cs) {
  const float x = Cvt<T>::to_f(src[e]);
  if (e >= rot_dims) return x;
  const float xp = Cvt<T>::to_f(src[e ^ 1]);
  const float2 c = cs[e >> 1];
  return (e & 1) ? x * c.x + xp * c.y : x * c.x - xp * c.y;
}

// Cache row of new token r: normed latent, rotated key part, zeros.  One warp.
template <typename T, int V>
__device__ __forceinline__ void ll_latent_row(const gb_ll_latent_args& a, int r) {
  const int lane = threadIdx.x & 31, b = r / a.n, pos = a.st[b].abs_pos + r - b * a.n;
  if (pos >= a.cap) return;
  const T* src = reinterpret_cast<const T*>(a.proj) + r * a.ld_proj + a.q_rank;
  T* dst = reinterpret_cast<T*>(a.cache) + ((long long)b * a.cap + pos) * a.ldc;
  auto get = [&](int i, float (&v)[V]) { ll_get(src + i, v); };
  ll_row_norm<32, V, 4>(a.rank, GB_LL_NORM_RMS, a.kv_norm, nullptr, a.eps, nullptr, get, get, [&](int i, const float (&v)[V]) { ll_put(dst + i, v); });
  const float2* cs = reinterpret_cast<const float2*>(a.cs) + (long long)r * (a.rot_dims / 2);
  for (int e = lane; e < a.ldc - a.rank; e += 32)
    dst[a.rank + e] = Cvt<T>::from_f(e < a.dr ? ll_turned(src + a.rank, e, a.rot_dims, cs) : 0.f);
}

// Two warps per row: one for the latent and the rotated part, one for the query latent.
template <typename T, int V>
__global__ void __launch_bounds__(256) ll_latent_store_kernel(const __grid_constant__ gb_ll_latent_args a) {
  pdl_wait();
  const int w = blockIdx.x * 8 + (threadIdx.x >> 5), r = w >> 1, lane = threadIdx.x & 31;
  if (r >= a.B * a.n) return;
  if (w & 1) {
    ll_latent_row<T, V>(a, r);
    return;
  }
  const T* src = reinterpret_cast<const T*>(a.proj) + r * a.ld_proj;
  T* dst = reinterpret_cast<T*>(a.cq) + r * a.ld_cq;
  auto get = [&](int i, float (&v)[V]) { ll_get(src + i, v); };
  ll_row_norm<32, V, 4>(a.q_rank, GB_LL_NORM_RMS, a.q_norm, nullptr, a.eps, nullptr, get, get, [&](int i, const float (&v)[V]) { ll_put(dst + i, v); });
  for (int i = a.q_rank + lane; i < a.ld_cq; i += 32) dst[i] = Cvt<T>::from_f(0.f);
}

// LPH lanes per (row, head), eight dimensions per lane (sizes in multiples of eight).
template <typename T, int LPH>
__global__ void __launch_bounds__(256) ll_latent_queries_vec_kernel(const __grid_constant__ gb_ll_latent_args a) {
  pdl_wait();
  const int lane = threadIdx.x & 31, c = (lane % LPH) * 8;
  const long long item = (blockIdx.x * 8LL + (threadIdx.x >> 5)) * (32 / LPH) + lane / LPH;
  if (item >= (long long)a.B * a.n * a.H || c >= a.dkp) return;
  const int r = (int)(item / a.H), h = (int)(item - (long long)r * a.H), dk = a.dn + a.dr;
  float v[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] = 0.f;
  if (c < dk) ll_load8(reinterpret_cast<const T*>(a.qc) + r * a.ld_qc + (long long)h * dk + c, v);
  const int t = c - a.dn;
  if (t >= 0 && t < a.rot_dims) {
    const float4* cs = reinterpret_cast<const float4*>(a.cs + (long long)r * a.rot_dims + t);
    const float4 p0 = cs[0], p1 = cs[1];
    const float cc[4] = {p0.x, p0.z, p1.x, p1.z}, sn[4] = {p0.y, p0.w, p1.y, p1.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float x = v[2 * e], y = v[2 * e + 1];
      v[2 * e] = x * cc[e] - y * sn[e];
      v[2 * e + 1] = y * cc[e] + x * sn[e];
    }
  }
  ll_store8(reinterpret_cast<T*>(a.q) + item * a.dkp + c, v);
}

// One warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) ll_latent_queries_kernel(const __grid_constant__ gb_ll_latent_args a) {
  pdl_wait();
  const long long item = blockIdx.x * 8LL + (threadIdx.x >> 5);
  if (item >= (long long)a.B * a.n * a.H) return;
  const int r = (int)(item / a.H), h = (int)(item - (long long)r * a.H), dk = a.dn + a.dr, lane = threadIdx.x & 31;
  const T* src = reinterpret_cast<const T*>(a.qc) + r * a.ld_qc + (long long)h * dk;
  T* dst = reinterpret_cast<T*>(a.q) + item * a.dkp;
  const float2* cs = reinterpret_cast<const float2*>(a.cs) + (long long)r * (a.rot_dims / 2);
  for (int e = lane; e < a.dkp; e += 32)
    dst[e] = e < a.dn ? src[e] : Cvt<T>::from_f(e < dk ? ll_turned(src + a.dn, e - a.dn, a.rot_dims, cs) : 0.f);
}

// grid (row groups, H [+ 1], runs of 256 columns): qa[r, h, :] = (key map of h)^T applied to the unrotated query, then its rotated
// part.  Eight warps share the sum over the query's dimensions; the first pieces of the map are requested before the wait for
// the kernel ahead.  Block row H, when there is one, writes the cache rows.
template <typename T, int V, int RB>
__global__ void __launch_bounds__(256) ll_latent_absorb_kernel(const __grid_constant__ gb_ll_latent_args a) {
  __shared__ float sq[RB][256];
  __shared__ __align__(16) float part[8][256];
  constexpr int PF = sizeof(T) == 4 ? 4 : 8;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, r0 = blockIdx.x * RB, nr = min(RB, a.B * a.n - r0), dk = a.dn + a.dr;
  const int c0 = blockIdx.z * 256, c = c0 + lane * 8;
  if (h == a.H) {
    pdl_wait();
    if (blockIdx.z == 0)
      for (int k = warp; k < nr; k += 8) ll_latent_row<T, V>(a, r0 + k);
    return;
  }
  const T* W = reinterpret_cast<const T*>(a.W_kv) + (long long)h * a.dkp * a.ld_w + c;
  LlRaw8<T> raw[PF];
#pragma unroll
  for (int i = 0; i < PF; ++i)
    if (c < a.rank && warp + 8 * i < a.dn) raw[i].load(W + (long long)(warp + 8 * i) * a.ld_w);
  pdl_wait();
  auto put = [&](int k, int col, float v) {
    const long long r = r0 + k;
    if (a.qa16) reinterpret_cast<T*>(a.qa16)[(r * a.heads_pad + h) * a.ld_qa16 + col] = Cvt<T>::from_f(v);
    else a.qa[(r * a.H + h) * a.ldc + col] = v;
  };
  for (int x = threadIdx.x; x < nr * dk; x += 256) {
    const int k = x / dk, e = x - k * dk, r = r0 + k;
    const T* src = reinterpret_cast<const T*>(a.qc) + r * a.ld_qc + (long long)h * dk;
    const float2* cs = reinterpret_cast<const float2*>(a.cs) + (long long)r * (a.rot_dims / 2);
    const float v = e < a.dn ? Cvt<T>::to_f(src[e]) : ll_turned(src + a.dn, e - a.dn, a.rot_dims, cs);
    sq[k][e] = v;
    if (e >= a.dn && blockIdx.z == 0) put(k, a.rank + e - a.dn, v);
  }
  __syncthreads();
  float acc[RB][8];
#pragma unroll
  for (int k = 0; k < RB; ++k)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[k][e] = 0.f;
  auto add = [&](int d, const LlRaw8<T>& x) {
    float w[8];
    x.expand(w);
#pragma unroll
    for (int k = 0; k < RB; ++k) {
      const float q = sq[k][d];
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[k][e] += q * w[e];
    }
  };
  if (c < a.rank) {
#pragma unroll
    for (int i = 0; i < PF; ++i)
      if (warp + 8 * i < a.dn) add(warp + 8 * i, raw[i]);
#pragma unroll 4
    for (int d = warp + 8 * PF; d < a.dn; d += 8) {
      LlRaw8<T> x;
      x.load(W + (long long)d * a.ld_w);
      add(d, x);
    }
  }
#pragma unroll
  for (int k = 0; k < RB; ++k) {
    if (k >= nr) break;
    if (k > 0) __syncthreads();
    ll_store8(&part[warp][8 * lane], acc[k]);
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) s += part[w][threadIdx.x];
    if (c0 + threadIdx.x < a.rank) put(k, c0 + threadIdx.x, s);
  }
}

template <typename T>
__device__ __forceinline__ float2 ll_pair(const T* p) {
  if constexpr (sizeof(T) == 4) return *reinterpret_cast<const float2*>(p);
  else return Cvt<T>::unpack2(*reinterpret_cast<const uint32_t*>(p));
}

// grid (rows * ceil(H / GQ), splits), 4 warps, GQ heads per block.  Lane l holds the pairs 2 (l + 32 k) of a stored row; each
// warp walks its keys with an online soft-max per head.
template <typename T, int NV, int GQ>
__global__ void __launch_bounds__(128) ll_latent_attn_kernel(const __grid_constant__ gb_ll_latent_args a) {
  pdl_wait();
  constexpr int KB = NV <= 3 ? 4 : 2, W = 64 * NV;            // keys in flight per warp
  const int chunks = (a.H + GQ - 1) / GQ;
  const int r = blockIdx.x / chunks, h0 = (blockIdx.x - r * chunks) * GQ, nh = min(GQ, a.H - h0), split = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, b = r / a.n;
  const int count = min(a.cap, a.st[b].abs_pos + r - b * a.n + 1), per = (count + a.splits - 1) / a.splits;
  const int lo = split * per, hi = min(count, lo + per), D = a.rank + a.dr;
  const T* rows = reinterpret_cast<const T*>(a.cache) + (long long)b * a.cap * a.ldc;
  float2 q[GQ][NV], o[GQ][NV];
  float m[GQ], l[GQ];
#pragma unroll
  for (int x = 0; x < GQ; ++x) {
    m[x] = -INFINITY; l[x] = 0.f;
    const float* qp = a.qa + ((long long)r * a.H + h0 + min(x, nh - 1)) * a.ldc;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = 2 * (lane + 32 * k);
      o[x][k] = make_float2(0.f, 0.f);
      q[x][k] = make_float2(c < D ? qp[c] * a.scale : 0.f, c + 1 < D ? qp[c + 1] * a.scale : 0.f);
    }
  }
  for (int e0 = lo + warp * KB; e0 < hi; e0 += 4 * KB) {
    float2 kf[KB][NV];
#pragma unroll
    for (int j = 0; j < KB; ++j) {
      const T* row = rows + (long long)min(e0 + j, hi - 1) * a.ldc;
#pragma unroll
      for (int k = 0; k < NV; ++k) {
        const int c = 2 * (lane + 32 * k);
        kf[j][k] = c < a.ldc ? ll_pair(row + c) : make_float2(0.f, 0.f);
      }
    }
#pragma unroll
    for (int x = 0; x < GQ; ++x) {
      float s[KB], mn = m[x];
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        s[j] = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) s[j] += q[x][k].x * kf[j][k].x + q[x][k].y * kf[j][k].y;
      }
#pragma unroll
      for (int d = 16; d > 0; d >>= 1)
#pragma unroll
        for (int j = 0; j < KB; ++j) s[j] += __shfl_xor_sync(0xffffffffu, s[j], d);
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        if (e0 + j >= hi) s[j] = -INFINITY;
        mn = fmaxf(mn, s[j]);
      }
      const float c = expf(m[x] - mn);              // the first key of a group is always real, so mn is finite
      l[x] *= c;
#pragma unroll
      for (int k = 0; k < NV; ++k) { o[x][k].x *= c; o[x][k].y *= c; }
#pragma unroll
      for (int j = 0; j < KB; ++j) {
        const float pr = expf(s[j] - mn);
        l[x] += pr;
#pragma unroll
        for (int k = 0; k < NV; ++k) { o[x][k].x += pr * kf[j][k].x; o[x][k].y += pr * kf[j][k].y; }
      }
      m[x] = mn;
    }
  }
  // the four warps' results, one head at a time
  __shared__ float sm_m[4][GQ], sm_l[4][GQ];
  __shared__ float2 sm_o[4][W / 2];
  if (lane == 0) {
#pragma unroll
    for (int x = 0; x < GQ; ++x) { sm_m[warp][x] = m[x]; sm_l[warp][x] = l[x]; }
  }
#pragma unroll
  for (int x = 0; x < GQ; ++x) {
    if (x >= nh) break;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < NV; ++k) sm_o[warp][lane + 32 * k] = o[x][k];
    __syncthreads();
    float mm = -INFINITY, ll = 0.f, f[4];
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, sm_m[w][x]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      f[w] = sm_m[w][x] == -INFINITY ? 0.f : expf(sm_m[w][x] - mm);
      ll += sm_l[w][x] * f[w];
    }
    const long long at = ((long long)r * a.H + h0 + x) * a.splits + split;
    float* dst = a.scratch + at * a.ldc;
    if (threadIdx.x == 0) {
      float* ml = a.scratch + (long long)a.B * a.n * a.H * a.splits * a.ldc + 2 * at;
      ml[0] = mm;
      ml[1] = ll;
    }
    for (int c = threadIdx.x; c < a.rank; c += 128) {
      const float* so = reinterpret_cast<const float*>(sm_o);
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) v += so[w * W + c] * f[w];
      dst[c] = v;
    }
  }
}

// A cluster of four blocks per (row, head): the splits' results, the head's value map, the output gate.  Each block combines a
// quarter of the latent dimensions (groups of threads take every g-th split), gives them to all four, and makes a quarter of
// the head's outputs; its first rows of the value map are requested before the wait for the kernel ahead.
constexpr int LM_THREADS = 512, LM_CL = 4;
template <typename T>
__global__ void __cluster_dims__(LM_CL, 1, 1) __launch_bounds__(LM_THREADS) ll_latent_merge_kernel(const __grid_constant__ gb_ll_latent_args a) {
  __shared__ float s_f[64];
  __shared__ __align__(16) float s_p[LM_THREADS * 4];
  __shared__ __align__(16) float s_o[1024];
  constexpr int WARPS = LM_THREADS / 32;
  const int item = blockIdx.x / LM_CL, rank = blockIdx.x % LM_CL, r = item / a.H, h = item - r * a.H, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int units = (a.rank + 7) / 8, mine = (2 * units + LM_CL - 1) / LM_CL;         // quads of dimensions per block
  const int ng = min(a.splits, LM_THREADS / mine), g = tid / mine, q = rank * mine + tid - g * mine;
  const bool works = g < ng && q < 2 * units;
  const long long at = ((long long)r * a.H + h) * a.splits;
  const float* base = a.scratch + at * a.ldc + 4 * q;
  const float* ml = a.scratch + (long long)a.B * a.n * a.H * a.splits * a.ldc + 2 * at;
  const T* W = reinterpret_cast<const T*>(a.W_kv) + ((long long)a.H * a.dkp + (long long)h * a.dvp) * a.ld_w;
  const int per = (a.dv + LM_CL - 1) / LM_CL, e_lo = rank * per + warp, e_hi = min(a.dv, (rank + 1) * per);
  constexpr int PW = 2;                                      // rows and pieces of 256 columns that are requested ahead
  LlRaw8<T> raw[PW][PW];
#pragma unroll
  for (int i = 0; i < PW; ++i)
#pragma unroll
    for (int k = 0; k < PW; ++k)
      if (e_lo + i * WARPS < e_hi && lane + 32 * k < units) raw[i][k].load(W + (long long)(e_lo + i * WARPS) * a.ld_w + (lane + 32 * k) * 8);
  pdl_wait();
  constexpr int AHEAD = 4;
  float4 v[AHEAD];
#pragma unroll
  for (int k = 0; k < AHEAD; ++k)
    if (works && g + k * ng < a.splits) v[k] = *reinterpret_cast<const float4*>(base + (long long)(g + k * ng) * a.ldc);
  if (warp == 0) {
    const float m0 = lane < a.splits ? ml[2 * lane] : -INFINITY, m1 = lane + 32 < a.splits ? ml[2 * lane + 64] : -INFINITY;
    const float l0 = lane < a.splits ? ml[2 * lane + 1] : 0.f, l1 = lane + 32 < a.splits ? ml[2 * lane + 65] : 0.f;
    const float mm = warp_max(fmaxf(m0, m1));
    const float f0 = m0 == -INFINITY ? 0.f : expf(m0 - mm), f1 = m1 == -INFINITY ? 0.f : expf(m1 - mm);
    const float l = warp_sum(l0 * f0 + l1 * f1), inv = l > 0.f ? 1.f / l : 0.f;
    s_f[lane] = f0 * inv;
    s_f[lane + 32] = f1 * inv;
  }
  cluster_sync_all();                                        // s_f is there, and the other blocks run
  if (g < ng) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    auto add = [&](int s, const float4& x) {
      const float f = s_f[s];
      if (f != 0.f) { o.x += x.x * f; o.y += x.y * f; o.z += x.z * f; o.w += x.w * f; }      // an empty split left nothing to read
    };
    if (works) {
#pragma unroll
      for (int k = 0; k < AHEAD; ++k)
        if (g + k * ng < a.splits) add(g + k * ng, v[k]);
#pragma unroll 4
      for (int s = g + AHEAD * ng; s < a.splits; s += ng) add(s, *reinterpret_cast<const float4*>(base + (long long)s * a.ldc));
    }
    *reinterpret_cast<float4*>(&s_p[tid * 4]) = o;
  }
  __syncthreads();
  for (int c = tid; c < 4 * mine; c += LM_THREADS) {
    const int dim = rank * 4 * mine + c;
    if (dim >= units * 8) break;
    float o = 0.f;
    if (dim < a.rank)
      for (int k = 0; k < ng; ++k) o += s_p[k * mine * 4 + c];
#pragma unroll
    for (int to = 0; to < LM_CL; ++to)
      asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(mapa_shared(smem_u32(&s_o[dim]), to)), "f"(o) : "memory");
  }
  cluster_sync_all();
  const T* gate = a.gate ? reinterpret_cast<const T*>(a.gate) + r * a.ld_gate + (long long)h * a.dv : nullptr;
  T* out = reinterpret_cast<T*>(a.out) + r * a.ldo + (long long)h * a.dv;
  auto dot = [&](const LlRaw8<T>& x, int u) {
    float w[8], o[8], s = 0.f;
    x.expand(w);
    ll_load8(&s_o[u * 8], o);
#pragma unroll
    for (int k = 0; k < 8; ++k) s += w[k] * o[k];
    return s;
  };
  auto finish = [&](int e, float s) {
    s = warp_sum(s);
    if (lane == 0) out[e] = Cvt<T>::from_f(gate ? s * ll_sigmoid(Cvt<T>::to_f(gate[e])) : s);
  };
  auto rest = [&](int e, int u0) {
    float s = 0.f;
    for (int u = u0; u < units; u += 32) {
      LlRaw8<T> x;
      x.load(W + (long long)e * a.ld_w + u * 8);
      s += dot(x, u);
    }
    return s;
  };
#pragma unroll
  for (int i = 0; i < PW; ++i) {
    const int e = e_lo + i * WARPS;
    if (e < e_hi) {
      float s = 0.f;
#pragma unroll
      for (int k = 0; k < PW; ++k)
        if (lane + 32 * k < units) s += dot(raw[i][k], lane + 32 * k);
      finish(e, s + rest(e, lane + 32 * PW));
    }
  }
  for (int e = e_lo + PW * WARPS; e < e_hi; e += WARPS) finish(e, rest(e, lane));
}

template <typename T>
static int ll_latent_attn_go(const gb_ll_latent_args& a, cudaStream_t st) {
  const int rows = a.B * a.n, D = a.ldc;
  if (a.qa16) {
    if (const int rc = gb_ll_latent_tc(&a, st)) return rc;
    GB_PDL_LAUNCH(ll_latent_merge_kernel<T>, dim3(rows * a.H * LM_CL), dim3(LM_THREADS), st, a);
    return gb_launch_rc();
  }
#define GO(NV, GQ) GB_PDL_LAUNCH((ll_latent_attn_kernel<T, NV, GQ>), dim3(rows * ((a.H + GQ - 1) / GQ), a.splits), dim3(128), st, a)
  if (D <= 128) GO(2, 4);
  else if (D <= 192) GO(3, 4);
  else if (D <= 320) GO(5, 4);
  else if (D <= 576) GO(9, 2);
  else GO(16, 1);
#undef GO
  GB_PDL_LAUNCH(ll_latent_merge_kernel<T>, dim3(rows * a.H * LM_CL), dim3(LM_THREADS), st, a);
  return gb_launch_rc();
}

}  // namespace gb

using namespace gb;

static uintptr_t ll_bits(const void* p) { return reinterpret_cast<uintptr_t>(p); }

static int ll_latent_check(const gb_ll_latent_args* p) {
  if (!p || !p->st || !p->cache || p->B <= 0 || p->n <= 0 || p->H <= 0 || p->dn <= 0 || p->dr <= 0 || p->dv <= 0 || p->rank <= 0 || p->q_rank <= 0) return -1;
  if (p->dn + p->dr > p->dkp || p->dv > p->dvp || p->dkp > 256 || p->dvp > 256 || p->dkp % 8 || p->dvp % 8) return -2;
  if (p->rot_dims < 0 || p->rot_dims % 2 || p->rot_dims > p->dr || (p->rot_dims > 0 && !p->cs)) return -3;
  if (p->ldc < p->rank + p->dr || p->ldc % 8 || p->ldc > 1024 || p->ld_w < p->ldc || p->ld_w % 8 || p->cap <= 0) return -4;
  if ((ll_bits(p->cache) | ll_bits(p->W_kv)) & 15) return -5;
  return p->dtype == 1 || p->dtype == 2 ? 0 : -6;
}

// eight values at a time: every piece of a projected row starts on sixteen bytes (32 for fp32)
static bool ll_latent_vec(const gb_ll_latent_args* p) {
  return p->q_rank % 8 == 0 && p->rank % 8 == 0 && p->ld_proj % 8 == 0 && ((ll_bits(p->proj) | ll_bits(p->cq) | ll_bits(p->q_norm) | ll_bits(p->kv_norm)) & 15) == 0 &&
         p->ld_cq % 8 == 0;
}

extern "C" int gb_ll_latent_store(const gb_ll_latent_args* p, cudaStream_t st) {
  if (const int rc = ll_latent_check(p)) return rc;
  if (!p->proj || !p->cq || !p->q_norm || !p->kv_norm || p->ld_cq < p->q_rank) return -1;
  const dim3 grid((p->B * p->n + 3) / 4);
  const bool vec = ll_latent_vec(p);
#define LS(T, V) GB_PDL_LAUNCH((ll_latent_store_kernel<T, V>), grid, dim3(256), st, *p)
  if (p->dtype == 1) { if (vec) LS(__nv_bfloat16, 8); else LS(__nv_bfloat16, 1); }
  else { if (vec) LS(float, 8); else LS(float, 1); }
#undef LS
  return gb_launch_rc();
}

extern "C" int gb_ll_latent_queries(const gb_ll_latent_args* p, cudaStream_t st) {
  if (const int rc = ll_latent_check(p)) return rc;
  if (!p->qc || !p->q) return -1;
  const long long items = (long long)p->B * p->n * p->H;
  if (p->dn % 8 == 0 && p->dr % 8 == 0 && p->rot_dims % 8 == 0 && p->ld_qc % 8 == 0 && ((ll_bits(p->qc) | ll_bits(p->q) | ll_bits(p->cs)) & 15) == 0) {
    const int lph = p->dkp <= 64 ? 8 : p->dkp <= 128 ? 16 : 32;
    const dim3 grid((unsigned)((items + 8 * (32 / lph) - 1) / (8 * (32 / lph))));
#define LQ(T, L) GB_PDL_LAUNCH((ll_latent_queries_vec_kernel<T, L>), grid, dim3(256), st, *p)
    if (p->dtype == 1) { if (lph == 8) LQ(__nv_bfloat16, 8); else if (lph == 16) LQ(__nv_bfloat16, 16); else LQ(__nv_bfloat16, 32); }
    else { if (lph == 8) LQ(float, 8); else if (lph == 16) LQ(float, 16); else LQ(float, 32); }
#undef LQ
    return gb_launch_rc();
  }
  const dim3 grid((unsigned)((items + 7) / 8));
  if (p->dtype == 1) GB_PDL_LAUNCH(ll_latent_queries_kernel<__nv_bfloat16>, grid, dim3(256), st, *p);
  else GB_PDL_LAUNCH(ll_latent_queries_kernel<float>, grid, dim3(256), st, *p);
  return gb_launch_rc();
}

extern "C" int gb_ll_latent_absorb(const gb_ll_latent_args* p, int store, cudaStream_t st) {
  if (const int rc = ll_latent_check(p)) return rc;
  if (!p->qc || (!p->qa && !p->qa16) || !p->W_kv || (p->qa16 && p->dtype != 1) || (store && (!p->proj || !p->kv_norm))) return -1;
  const int rows = p->B * p->n, rb = rows > 1 ? 4 : 1;
  const bool vec = ll_latent_vec(p);
  const dim3 grid((rows + rb - 1) / rb, p->H + (store ? 1 : 0), (p->rank + 255) / 256);
#define LA(T, V) do { if (rb == 1) GB_PDL_LAUNCH((ll_latent_absorb_kernel<T, V, 1>), grid, dim3(256), st, *p); \
                      else GB_PDL_LAUNCH((ll_latent_absorb_kernel<T, V, 4>), grid, dim3(256), st, *p); } while (0)
  if (p->dtype == 1) { if (vec) LA(__nv_bfloat16, 8); else LA(__nv_bfloat16, 1); }
  else { if (vec) LA(float, 8); else LA(float, 1); }
#undef LA
  return gb_launch_rc();
}

extern "C" int gb_ll_latent_attn(const gb_ll_latent_args* p, cudaStream_t st) {
  if (const int rc = ll_latent_check(p)) return rc;
  if ((!p->qa && !p->qa16) || (p->qa16 && p->dtype != 1) || !p->W_kv || !p->out || !p->scratch || p->splits < 1 || p->splits > 64) return -1;
  return p->dtype == 1 ? ll_latent_attn_go<__nv_bfloat16>(*p, st) : ll_latent_attn_go<float>(*p, st);
}
