// Prompt attention of layer-list models on the tensor cores (interface in gb_layers.h): queries of the new tokens against
// the layer's cache (kept first positions + ring), bf16 operands, fp32 scores, weights and sums.
//
// Work split as in attention_tc.cu: warp 4 = TMA producer, warp 5 = MMA issuer, warps 0-3 = one soft-max thread per query
// row; persistent CTAs walk (query tile, sequence, head) items from the longest on.  What differs is where keys come
// from: an item's key tiles are the tiles of the kept prefix (rows 0 .. keep of the cache) followed by the ring tiles
// that overlap its window.  The ring is a multiple of 128 rows long and starts at row `keep`, so a tile of 128
// consecutive positions is 128 consecutive rows.  The item ends with the sink in the denominator and the output gate.
//
// CAPPED: scores pass through cap * tanh(. / cap), less slope * distance.  They are then at most cap, and at least -cap on
// the query's own place, so exponentials need no running maximum: one pass over the scores, nothing to rescale.
#include <algorithm>

#include "sm100_common.cuh"
#include "gb_layers.h"
#include "tc_tiles.cuh"
#include "layers_util.cuh"

namespace gb {

constexpr int LA_THREADS = 192;

__device__ __forceinline__ float ll_ex2(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

constexpr float LA_CAP_MAX = 60.f;          // e^+-cap and sums of many such terms stay well inside fp32's range

__device__ __forceinline__ float ll_rcp(float x) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

template <int DK, int DV, bool CAPPED>
__global__ void __launch_bounds__(LA_THREADS) ll_attn_tc_kernel(const __grid_constant__ CUtensorMap tmQ,
                                                                const __grid_constant__ CUtensorMap tmK,
                                                                const __grid_constant__ CUtensorMap tmV,
                                                                const __grid_constant__ gb_ll_attn_args a) {
  using T = __nv_bfloat16;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  constexpr uint32_t TQ = AT_M * DK * 2, TV = AT_N * DV * 2;
  uint8_t* smem;
  if constexpr (DK == 64 && DV == 64) {      // 112 KB and a few bytes: two CTAs per SM, no slack to align by hand
    if (smem_u32(smem_raw) & 1023u) {
      if (threadIdx.x == 0) atomicCAS(a.status, 0, ST_BAD_ARGUMENT);
      return;
    }
    smem = smem_raw;
  } else {
    smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  }
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + TQ;              // 2 stages
  uint8_t* sV = sK + 2 * TQ;          // 2 stages
  uint8_t* sP = sV + 2 * TV;          // [128 x 128] 16-bit
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + AT_M * AT_N * 2);
  uint64_t* q_full = bars;            // 1
  uint64_t* kv_full = bars + 1;       // 2
  uint64_t* kv_empty = bars + 3;      // 2
  uint64_t* s_full = bars + 5;
  uint64_t* p_ready = bars + 6;
  uint64_t* o_full = bars + 7;
  uint64_t* q_empty = bars + 8;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 9);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_qt = (a.n + AT_M - 1) / AT_M, BH = a.B * a.H, n_items = n_qt * BH, rep = a.H / a.G;
  const int ring = a.cap - a.keep;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(q_empty, 1);
    for (int s = 0; s < 2; ++s) { mbar_init(&kv_full[s], 1); mbar_init(&kv_empty[s], 1); }
    mbar_init(s_full, 1);
    mbar_init(p_ready, 4);
    mbar_init(o_full, 1);
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 5) { tmem_alloc(tmem_slot, 256); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_S = tmem_base, tmem_O = tmem_base + AT_N;

  // n_kt tiles of the kept prefix, then ring tiles r_lo .. r_lo + n_rt - 1 (tile i: positions keep + 128 i ...)
  struct Item { int b, h, q0, p0, n_kt, r_lo, n_rt; };
  auto item_of = [&](int item) {
    Item it;
    const int zt = item / BH, bh = item - zt * BH;
    it.b = bh / a.H;
    it.h = bh - it.b * a.H;
    it.q0 = (n_qt - 1 - zt) * AT_M;
    it.p0 = a.st[it.b].abs_pos;
    const int first = it.p0 + it.q0, last = it.p0 + min(a.n, it.q0 + AT_M) - 1;
    it.n_kt = (min(a.keep, last + 1) + AT_N - 1) / AT_N;
    const int lo = max(a.keep, a.window > 0 ? first - a.window + 1 : 0);
    it.r_lo = (lo - a.keep) / AT_N;
    it.n_rt = last < lo ? 0 : (last - a.keep) / AT_N - it.r_lo + 1;
    return it;
  };
  auto tile_row = [&](const Item& it, int t) {          // first cache row of the item's key tile t
    return it.b * a.cap + (t < it.n_kt ? t * AT_N : a.keep + (int)(((long long)(it.r_lo + t - it.n_kt) * AT_N) % ring));
  };

  auto tile_pos = [&](const Item& it, int t) {          // position of that row
    return t < it.n_kt ? t * AT_N : a.keep + (it.r_lo + t - it.n_kt) * AT_N;
  };

  if (warp == 4) {
    if (lane == 0) {
      uint32_t kv_it = 0, q_it = 0;
      bool ok = true;
      for (int item = blockIdx.x; item < n_items && ok; item += gridDim.x, ++q_it) {
        const Item it = item_of(item);
        if (!at_wait(q_empty, (q_it & 1u) ^ 1u, a.status, ST_TIMEOUT_EMPTY, abort_flag)) break;
        mbar_arrive_expect_tx(q_full, TQ);
        load_tile<DK>(&tmQ, q_full, sQ, it.h * DK, it.b * a.n + it.q0);
        const int g = it.h / rep;
        for (int t = 0; t < it.n_kt + it.n_rt; ++t, ++kv_it) {
          const int s = kv_it & 1, ph = (kv_it >> 1) & 1;
          if (!at_wait(&kv_empty[s], ph ^ 1, a.status, ST_TIMEOUT_EMPTY, abort_flag)) { ok = false; break; }
          mbar_arrive_expect_tx(&kv_full[s], TQ + TV);
          const int row = tile_row(it, t);
          load_tile<DK>(&tmK, &kv_full[s], sK + s * TQ, g * DK, row);
          load_tile<DV>(&tmV, &kv_full[s], sV + s * TV, g * DV, row);
        }
      }
    }
    __syncwarp();
  } else if (warp == 5) {
    if (lane == 0) {
      const uint32_t idesc_s = make_idesc_f16(1, 0, 0, AT_M, AT_N);
      const uint32_t idesc_o = make_idesc_f16(1, 0, 1, AT_M, DV);
      uint32_t kv_it = 0, q_it = 0;
      bool ok = true;
      for (int item = blockIdx.x; item < n_items && ok; item += gridDim.x, ++q_it) {
        const Item it = item_of(item);
        const int n_tiles = it.n_kt + it.n_rt;
        if (!at_wait(q_full, q_it & 1u, a.status, ST_TIMEOUT_FULL, abort_flag)) break;
        for (int t = 0; t < n_tiles; ++t, ++kv_it) {
          const int s = kv_it & 1, ph = (kv_it >> 1) & 1;
          if (!at_wait(&kv_full[s], ph, a.status, ST_TIMEOUT_FULL, abort_flag)) { ok = false; break; }
          tc_fence_after();
          mma_kmajor_kmajor<DK>(tmem_S, smem_u32(sQ), smem_u32(sK + s * TQ), idesc_s, false);
          umma_commit(s_full);
          if (t == n_tiles - 1) umma_commit(q_empty);
          if (!at_wait(p_ready, kv_it & 1u, a.status, ST_TIMEOUT_TMEM_EMPTY, abort_flag)) { ok = false; break; }
          tc_fence_after();
          mma_kmajor_mnmajor<AT_N>(tmem_O, smem_u32(sP), smem_u32(sV + s * TV), idesc_o, t > 0);
          umma_commit(o_full);
          umma_commit(&kv_empty[s]);
        }
      }
    }
    __syncwarp();
  } else {
    const int r = threadIdx.x;
    const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
    const float sc2 = a.scale * 1.4426950408889634f;
    // tanh(z) = 1 - 2 / (e^2z + 1): the exponent's factor, and cap in log2 units
    const float cap_in = CAPPED ? 2.f * sc2 / a.softcap : 0.f, cap2 = a.softcap * 1.4426950408889634f;
    uint32_t tile_it = 0;
    bool ok = true;
    for (int item = blockIdx.x; item < n_items && ok; item += gridDim.x) {
      const Item it = item_of(item);
      const int i = it.p0 + it.q0 + r, i_first = it.p0 + it.q0, i_last = it.p0 + min(a.n, it.q0 + AT_M) - 1;
      const bool row_ok = it.q0 + r < a.n;
      float m2 = CAPPED ? 0.f : -INFINITY, l = 0.f;            // maximum in use (log2 units) and the row sum against it
      const float slope2 = CAPPED && a.slopes ? a.slopes[it.h] * 1.4426950408889634f : 0.f;
      for (int t = 0; t < it.n_kt + it.n_rt; ++t, ++tile_it) {
        // visible columns of this tile: lo .. hi
        int lo, hi;
        bool need_mask;
        if (t < it.n_kt) {
          lo = 0;
          hi = min(i, a.keep - 1) - t * AT_N;
          need_mask = true;
        } else {
          const int base = a.keep + (it.r_lo + t - it.n_kt) * AT_N;
          lo = a.window > 0 ? i - a.window + 1 - base : 0;
          hi = i - base;
          need_mask = base + AT_N - 1 > i_first || (a.window > 0 && i_last - a.window + 1 > base);
        }
        if (!at_wait(s_full, tile_it & 1u, a.status, ST_TIMEOUT_TMEM_FULL, abort_flag)) { ok = false; break; }
        tc_fence_after();
        if constexpr (!CAPPED) {
          float mr[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll 1
          for (int c = 0; c < AT_N / 32; ++c) {
            uint32_t rg[32];
            tmem_ld_32x32(tmem_S + lane_base + c * 32, rg);
            tmem_ld_wait();
            if (!need_mask) {
#pragma unroll
              for (int k = 0; k < 32; ++k) mr[k & 3] = fmaxf(mr[k & 3], __uint_as_float(rg[k]));
            } else {
#pragma unroll
              for (int k = 0; k < 32; ++k) {
                const int j = c * 32 + k;
                if (j <= hi && j >= lo) mr[k & 3] = fmaxf(mr[k & 3], __uint_as_float(rg[k]));
              }
            }
          }
          float mt = fmaxf(fmaxf(mr[0], mr[1]), fmaxf(mr[2], mr[3])) * sc2;
          if (!row_ok) mt = 0.f;
          const bool grow = mt > m2 + 8.f || (m2 == -INFINITY && mt != -INFINITY);
          if (__any_sync(0xffffffffu, grow)) {
            const float m_new = fmaxf(m2, mt);
            if (t > 0) {
              const float corr = (m2 == -INFINITY) ? 1.f : ll_ex2(m2 - m_new);
              l *= corr;
              if (!at_wait(o_full, (tile_it - 1u) & 1u, a.status, ST_TIMEOUT_TMEM_FULL, abort_flag)) { ok = false; break; }
              tc_fence_after();
#pragma unroll
              for (int c = 0; c < DV / 16; ++c) {
                uint32_t rg[16];
                tmem_ld_32x16(tmem_O + lane_base + c * 16, rg);
                tmem_ld_wait();
#pragma unroll
                for (int k = 0; k < 16; ++k) rg[k] = __float_as_uint(__uint_as_float(rg[k]) * corr);
                tmem_st_32x16(tmem_O + lane_base + c * 16, rg);
              }
              tmem_st_wait();
            }
            m2 = m_new;
          }
        }
        float ls[2] = {0.f, 0.f};
        const bool dead = m2 == -INFINITY || !row_ok;
        const float near2 = CAPPED ? cap2 - slope2 * (float)(i - tile_pos(it, t)) : 0.f;     // cap less the bias, at the tile's column 0
#pragma unroll 1
        for (int c = 0; c < AT_N / 32; ++c) {
          uint32_t rg[32];
          tmem_ld_32x32(tmem_S + lane_base + c * 32, rg);
          tmem_ld_wait();
          float pv[32];
          if constexpr (CAPPED) {
            const float near_c = near2 + slope2 * (float)(c * 32);
#pragma unroll
            for (int k = 0; k < 32; ++k) {
              const float th = ll_rcp(1.f + ll_ex2(__uint_as_float(rg[k]) * cap_in));
              const float e = ll_ex2(fmaf(-2.f * cap2, th, fmaf(slope2, (float)k, near_c)));
              pv[k] = e;
            }
            if (need_mask) {
#pragma unroll
              for (int k = 0; k < 32; ++k)
                if (dead || c * 32 + k > hi || c * 32 + k < lo) pv[k] = 0.f;
            }
#pragma unroll
            for (int k = 0; k < 32; ++k) ls[k & 1] += pv[k];
          } else if (!need_mask) {
#pragma unroll
            for (int k = 0; k < 32; ++k) {
              const float e = ll_ex2(fmaf(__uint_as_float(rg[k]), sc2, -m2));
              pv[k] = e;
              ls[k & 1] += e;
            }
          } else {
#pragma unroll
            for (int k = 0; k < 32; ++k) {
              const int j = c * 32 + k;
              const float e = (!dead && j <= hi && j >= lo) ? ll_ex2(fmaf(__uint_as_float(rg[k]), sc2, -m2)) : 0.f;
              pv[k] = e;
              ls[k & 1] += e;
            }
          }
          store_p_chunk<T>(sP, r, c * 32, pv);
        }
        l += ls[0] + ls[1];
        tc_fence_before();
        fence_proxy_async();
        __syncwarp();
        if (lane == 0) mbar_arrive(p_ready);
      }
      if (!ok) break;
      if (!at_wait(o_full, (tile_it - 1u) & 1u, a.status, ST_TIMEOUT_TMEM_FULL, abort_flag)) { ok = false; break; }
      tc_fence_after();
      float fac = 1.f;
      if (a.sink) {
        const float sk = a.sink[it.h] * 1.4426950408889634f, mn = fmaxf(m2, sk);
        fac = ll_ex2(m2 - mn);
        l = l * fac + ll_ex2(sk - mn);
      }
      fac = l > 0.f ? fac / l : 0.f;
      const long long row = (long long)it.b * a.n + it.q0 + r;
      T* op = reinterpret_cast<T*>(a.out) + row * a.ldo + it.h * a.dv;
      const T* gp = reinterpret_cast<const T*>(a.gate) + row * a.ld_gate + it.h * a.dv;
      const bool vec = a.dv == DV && ((reinterpret_cast<uintptr_t>(op) | reinterpret_cast<uintptr_t>(gp)) & 15) == 0;
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t rg[32];
        tmem_ld_32x32(tmem_O + lane_base + c * 32, rg);
        tmem_ld_wait();
        if (row_ok && vec) {
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            float v[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = __uint_as_float(rg[8 * k + e]) * fac;
            if (a.gate) {
              const uint4 gq = reinterpret_cast<const uint4*>(gp)[c * 4 + k];
              const uint32_t gw[4] = {gq.x, gq.y, gq.z, gq.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const float2 z = Cvt<T>::unpack2(gw[e]);
                v[2 * e] *= __fdividef(1.f, 1.f + ll_ex2(-1.4426950408889634f * z.x));
                v[2 * e + 1] *= __fdividef(1.f, 1.f + ll_ex2(-1.4426950408889634f * z.y));
              }
            }
            uint4 q;
            q.x = Cvt<T>::pack2(v[0], v[1]); q.y = Cvt<T>::pack2(v[2], v[3]);
            q.z = Cvt<T>::pack2(v[4], v[5]); q.w = Cvt<T>::pack2(v[6], v[7]);
            reinterpret_cast<uint4*>(op)[c * 4 + k] = q;
          }
        } else if (row_ok) {
#pragma unroll
          for (int k = 0; k < 32; ++k) {
            const int e = c * 32 + k;
            if (e < a.dv) {
              float v = __uint_as_float(rg[k]) * fac;
              if (a.gate) v *= ll_sigmoid(Cvt<T>::to_f(gp[e]));
              op[e] = Cvt<T>::from_f(v);
            }
          }
        }
        __syncwarp();                       // the next tensor-memory load is the whole warp's
      }
      tc_fence_before();
    }
  }
  __syncthreads();
  if (*abort_flag) {
    for (int k = 0; k < 64; ++k) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 5) { tc_fence_after(); tmem_dealloc(tmem_base, 256); }
}

template <int DK, int DV, bool CAPPED>
static int ll_attn_tc_go(const gb_ll_attn_args& a, cudaStream_t st) {
  CUtensorMap tq, tk, tv;
  const uint64_t rows = (uint64_t)a.B * a.n, crows = (uint64_t)a.B * a.cap;
  if (gb_make_tmap_2d_16b(&tq, a.q, rows, (uint64_t)a.H * DK, (uint64_t)a.H * DK, AT_M, 64, 1)) return -20;
  if (gb_make_tmap_2d_16b(&tk, a.cache_k, crows, (uint64_t)a.G * DK, (uint64_t)a.ld_k, AT_N, 64, 1)) return -21;
  if (gb_make_tmap_2d_16b(&tv, a.cache_v, crows, (uint64_t)a.G * DV, (uint64_t)a.ld_v, AT_N, 64, 1)) return -22;
  constexpr bool pair = DK == 64 && DV == 64;
  constexpr size_t smem = (size_t)AT_M * DK * 2 * 3 + (size_t)AT_N * DV * 2 * 2 + AT_M * AT_N * 2 + 128 + (pair ? 0 : 1024);
  auto kern = ll_attn_tc_kernel<DK, DV, CAPPED>;
  static int sms = 0;
  if (!sms) {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) return -10;
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return -10;
    (void)cudaFuncSetAttribute(kern, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
  }
  const long long items = (long long)((a.n + AT_M - 1) / AT_M) * a.B * a.H;
  if (items > 0x7fffffffll - 1024) return -1;
  kern<<<(unsigned)std::min<long long>(items, (pair ? 2ll : 1ll) * sms), LA_THREADS, smem, st>>>(tq, tk, tv, a);
  return gb_launch_rc();
}

template <bool CAPPED>
static int ll_attn_tc_sizes(const gb_ll_attn_args& a, cudaStream_t st) {
  if (a.dkp == 64) return a.dvp == 64 ? ll_attn_tc_go<64, 64, CAPPED>(a, st) : ll_attn_tc_go<64, 128, CAPPED>(a, st);
  return a.dvp == 64 ? ll_attn_tc_go<128, 64, CAPPED>(a, st) : ll_attn_tc_go<128, 128, CAPPED>(a, st);
}

}  // namespace gb

using namespace gb;

extern "C" int gb_ll_attn_tc_ok(const gb_ll_attn_args* p) {
  if (!p || p->dtype != 1) return -1;
  if ((p->dkp != 64 && p->dkp != 128) || (p->dvp != 64 && p->dvp != 128)) return -2;
  if (p->softcap > 0.f ? p->softcap > LA_CAP_MAX : p->slopes != nullptr) return -3;
  if (!(p->softcap > 0.f) && !(p->scale > 0.f)) return -3;          // the row maximum is taken on raw scores
  if (p->ld_k % 8 || p->ld_v % 8 || p->ld_k < p->G * p->dkp || p->ld_v < p->G * p->dvp) return -4;
  if (p->cap <= p->keep || (p->cap - p->keep) % AT_N) return -4;
  if ((long long)p->B * p->cap > 0x7fffffffll || (long long)p->B * p->n > 0x7fffffffll) return -5;
  return 0;
}

extern "C" int gb_ll_attn_tc(const gb_ll_attn_args* p, cudaStream_t st) {
  if (const int rc = gb_ll_attn_tc_ok(p)) return rc;
  if (!p->q || !p->cache_k || !p->cache_v || !p->out || !p->st || !p->status || p->B <= 0 || p->n <= 0 || p->H % p->G) return -1;
  return p->softcap > 0.f ? ll_attn_tc_sizes<true>(*p, st) : ll_attn_tc_sizes<false>(*p, st);
}
