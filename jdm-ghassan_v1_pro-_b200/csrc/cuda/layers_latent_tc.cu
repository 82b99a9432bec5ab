// Attention of a few new tokens over stored latents on the tensor cores (interface in gb_layers.h), bf16.
//
// All heads read the same rows, so one tile of 128 rows [128 keys x (rank + dr)], fetched once by TMA, is both operands'
// source: scores are S^T = rows * Q^T (keys along the accumulator's lanes, heads along its columns: 16 or 32 columns instead
// of 128 padded query rows), and outputs are O^T += rows^T * P^T, the same bytes read with the latent dimensions as the M
// extent.  A CTA takes a run of tiles of one token and one group of heads and leaves a partial result; warp 4 fetches, warp 5
// issues, warps 0-3 are one thread per key.
#include "sm100_common.cuh"
#include "gb_layers.h"
#include "layers_util.cuh"
#include "tc_tiles.cuh"

namespace gb {

constexpr int LT_THREADS = 192;
constexpr int LT_BAR_BYTES = 256;
constexpr size_t LT_SMEM_MAX = 227 * 1024;

__device__ __forceinline__ float lt_ex2(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
__device__ __forceinline__ void lt_keys_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }      // warps 0-3

template <int HP>
__device__ __forceinline__ void lt_tmem_load(uint32_t addr, uint32_t (&r)[HP]) {
  if constexpr (HP == 32) tmem_ld_32x32(addr, r);
  else tmem_ld_32x16(addr, r);
  tmem_ld_wait();
}

// Reduction of HP values per lane over the warp's lanes; lane l returns that of value l % HP.
template <int HP, typename F>
__device__ __forceinline__ float lt_transpose_reduce(const float (&v)[HP], F f) {
  const int lane = threadIdx.x & 31;
  float t[HP];
#pragma unroll
  for (int i = 0; i < HP; ++i) t[i] = v[i];
#pragma unroll
  for (int o = HP / 2; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? t[i] : t[i + o], own = up ? t[i + o] : t[i];
      t[i] = f(own, __shfl_xor_sync(0xffffffffu, send, o));
    }
  }
  if constexpr (HP == 16) t[0] = f(t[0], __shfl_xor_sync(0xffffffffu, t[0], 16));
  return t[0];
}

template <int HP>
__global__ void __launch_bounds__(LT_THREADS) ll_latent_tc_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmQ,
                                                                  const __grid_constant__ gb_ll_latent_args a, int panels, int stages) {
  using T = __nv_bfloat16;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr uint32_t KP = AT_N * 128, QP = HP * 128;             // bytes of a 64-column panel of keys, of queries
  uint8_t* sK = smem;
  uint8_t* sQ = sK + (size_t)stages * panels * KP;
  uint8_t* sP = sQ + panels * QP;                                // [HP heads x 128 keys], two panels
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + 2 * QP);
  uint64_t* q_full = bars;
  uint64_t* kv_full = bars + 1;                                  // 2
  uint64_t* kv_empty = bars + 3;                                 // 2
  uint64_t* s_full = bars + 5;
  uint64_t* p_ready = bars + 6;
  uint64_t* o_full = bars + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  __shared__ __align__(16) float s_red[4][HP], s_m[HP], s_corr[HP];
  __shared__ int s_grow;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int groups = a.heads_pad / HP, r = blockIdx.x / groups, h0 = (blockIdx.x - r * groups) * HP, b = r / a.n, split = blockIdx.y;
  const int chunks = (a.rank + 127) / 128, dsteps = (a.rank + a.dr + 15) / 16;
  const uint32_t cols = HP * (1 + chunks) <= 64 ? 64 : HP * (1 + chunks) <= 128 ? 128 : 256;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < 2; ++s) { mbar_init(&kv_full[s], 1); mbar_init(&kv_empty[s], 1); }
    mbar_init(s_full, 1);
    mbar_init(p_ready, 4);
    mbar_init(o_full, 1);
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 4 && lane == 0) { tma_prefetch_desc(&tmC); tma_prefetch_desc(&tmQ); }
  pdl_wait();
  if (warp == 5) { tmem_alloc(tmem_slot, cols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_S = *tmem_slot, tmem_O = tmem_S + HP;

  const int count = min(a.cap, a.st[b].abs_pos + r - b * a.n + 1), tiles = (count + AT_N - 1) / AT_N, per = (tiles + a.splits - 1) / a.splits;
  const int t_lo = split * per, n_t = max(0, min(tiles, t_lo + per) - t_lo);

  if (warp == 4) {
    if (lane == 0 && n_t > 0) {
      mbar_arrive_expect_tx(q_full, panels * QP);
      for (int p = 0; p < panels; ++p) tma_load_2d(&tmQ, q_full, sQ + p * QP, p * 64, r * a.heads_pad + h0);
      for (int t = 0; t < n_t; ++t) {
        const int s = t % stages, ph = (t / stages) & 1;
        if (!at_wait(&kv_empty[s], ph ^ 1, a.status, ST_TIMEOUT_EMPTY, abort_flag)) break;
        mbar_arrive_expect_tx(&kv_full[s], panels * KP);
        for (int p = 0; p < panels; ++p)
          tma_load_2d(&tmC, &kv_full[s], sK + (size_t)(s * panels + p) * KP, p * 64, b * a.cap + (t_lo + t) * AT_N);
      }
    }
    __syncwarp();
  } else if (warp == 5) {
    if (lane == 0 && n_t > 0) {
      const uint32_t idesc_s = make_idesc_f16(1, 0, 0, AT_N, HP), idesc_o = make_idesc_f16(1, 1, 0, 128, HP);
      const uint64_t dq0 = make_smem_desc_sw128(smem_u32(sQ), 16, 1024), dp0 = make_smem_desc_sw128(smem_u32(sP), 16, 1024);
      bool ok = at_wait(q_full, 0, a.status, ST_TIMEOUT_FULL, abort_flag);
      for (int t = 0; t < n_t && ok; ++t) {
        const int s = t % stages, ph = (t / stages) & 1;
        if (!at_wait(&kv_full[s], ph, a.status, ST_TIMEOUT_FULL, abort_flag)) break;
        tc_fence_after();
        // descriptors step by whole panels (start addresses count 16 bytes): one thread issues, so few instructions per product
        const uint32_t k0 = smem_u32(sK + (size_t)s * panels * KP);
        uint64_t dk = make_smem_desc_sw128(k0, 16, 1024), dq = dq0;
        for (int kk = 0; kk < dsteps; kk += 4, dk += KP >> 4, dq += QP >> 4) {
          const int left = dsteps - kk;
          umma_f16(tmem_S, dk, dq, idesc_s, kk > 0);
          if (left > 1) umma_f16(tmem_S, dk + 2, dq + 2, idesc_s, 1);
          if (left > 2) umma_f16(tmem_S, dk + 4, dq + 4, idesc_s, 1);
          if (left > 3) umma_f16(tmem_S, dk + 6, dq + 6, idesc_s, 1);
        }
        umma_commit(s_full);
        if (!at_wait(p_ready, t & 1, a.status, ST_TIMEOUT_TMEM_EMPTY, abort_flag)) break;
        tc_fence_after();
        uint64_t dv = make_smem_desc_sw128(k0, KP, 1024);
        for (int c = 0; c < chunks; ++c, dv += 2 * (KP >> 4))
#pragma unroll
          for (int kk = 0; kk < AT_N / 16; ++kk)      // A: latent dimensions along M (two panels), keys along K, 16 rows a step
            umma_f16(tmem_O + c * HP, dv + kk * (2048 >> 4), dp0 + ((kk >> 2) * QP + (kk & 3) * 32) / 16, idesc_o, (t > 0 || kk > 0) ? 1u : 0u);
        umma_commit(&kv_empty[s]);
        umma_commit(o_full);
      }
    }
    __syncwarp();
  } else if (n_t > 0) {
    // a wait that runs out does not leave the loop: the four warps meet at the same barriers
    const int key = threadIdx.x;
    const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
    const float sc2 = a.scale * 1.4426950408889634f;
    bool ok = true;
    float lsum[HP];
#pragma unroll
    for (int h = 0; h < HP; ++h) lsum[h] = 0.f;
    if (threadIdx.x < HP) s_m[threadIdx.x] = -INFINITY;
    for (int t = 0; t < n_t; ++t) {
      if (ok && !at_wait(s_full, t & 1, a.status, ST_TIMEOUT_TMEM_FULL, abort_flag)) ok = false;
      if (ok && t > 0 && !at_wait(o_full, (t - 1) & 1, a.status, ST_TIMEOUT_TMEM_FULL, abort_flag)) ok = false;
      __syncwarp();
      tc_fence_after();
      float s[HP];
      {
        uint32_t rg[HP];
        lt_tmem_load<HP>(tmem_S + lane_base, rg);
        const bool seen = (t_lo + t) * AT_N + key < count;
#pragma unroll
        for (int h = 0; h < HP; ++h) s[h] = seen ? __uint_as_float(rg[h]) * sc2 : -INFINITY;
      }
      const float top = lt_transpose_reduce<HP>(s, [](float x, float y) { return fmaxf(x, y); });
      if (lane < HP) s_red[warp][lane] = top;
      lt_keys_sync();
      if (warp == 0) {
        bool grow = false;
        if (lane < HP) {
          const float mt = fmaxf(fmaxf(s_red[0][lane], s_red[1][lane]), fmaxf(s_red[2][lane], s_red[3][lane])), mo = s_m[lane];
          grow = mt > mo + 8.f || (mo == -INFINITY && mt != -INFINITY);
          s_corr[lane] = grow && mo != -INFINITY ? lt_ex2(mo - mt) : 1.f;
          if (grow) s_m[lane] = mt;
        }
        const bool any = __any_sync(0xffffffffu, grow);
        if (lane == 0) s_grow = any;
      }
      lt_keys_sync();
      if (t > 0 && s_grow) {
        float corr[HP];
#pragma unroll
        for (int h = 0; h < HP; h += 4) {
          const float4 q = *reinterpret_cast<const float4*>(&s_corr[h]);
          corr[h] = q.x; corr[h + 1] = q.y; corr[h + 2] = q.z; corr[h + 3] = q.w;
        }
#pragma unroll
        for (int h = 0; h < HP; ++h) lsum[h] *= corr[h];
        for (int c = 0; c < chunks; ++c)
#pragma unroll
          for (int p = 0; p < HP / 16; ++p) {
            uint32_t rg[16];
            tmem_ld_32x16(tmem_O + lane_base + c * HP + p * 16, rg);
            tmem_ld_wait();
#pragma unroll
            for (int k = 0; k < 16; ++k) rg[k] = __float_as_uint(__uint_as_float(rg[k]) * corr[p * 16 + k]);
            tmem_st_32x16(tmem_O + lane_base + c * HP + p * 16, rg);
          }
        tmem_st_wait();
      }
#pragma unroll
      for (int h = 0; h < HP; h += 4) {
        const float4 q = *reinterpret_cast<const float4*>(&s_m[h]);
        s[h] = lt_ex2(s[h] - q.x); s[h + 1] = lt_ex2(s[h + 1] - q.y); s[h + 2] = lt_ex2(s[h + 2] - q.z); s[h + 3] = lt_ex2(s[h + 3] - q.w);
      }
      uint8_t* panel = sP + (key >> 6) * QP;
#pragma unroll
      for (int h = 0; h < HP; ++h) {
        lsum[h] += s[h];
        *reinterpret_cast<T*>(panel + sw128_off(h, key & 63)) = Cvt<T>::from_f(s[h]);
      }
      tc_fence_before();
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    const float tot = lt_transpose_reduce<HP>(lsum, [](float x, float y) { return x + y; });
    if (lane < HP) s_red[warp][lane] = tot;
    lt_keys_sync();
    const long long first = ((long long)r * a.H + h0) * a.splits + split;
    if (threadIdx.x < HP && h0 + threadIdx.x < a.H) {
      const int h = threadIdx.x;
      float* ml = a.scratch + (long long)a.B * a.n * a.H * a.splits * a.ldc + 2 * (first + (long long)h * a.splits);
      ml[0] = s_m[h] * 0.6931471805599453f;
      ml[1] = s_red[0][h] + s_red[1][h] + s_red[2][h] + s_red[3][h];
    }
    if (ok && !at_wait(o_full, (n_t - 1) & 1, a.status, ST_TIMEOUT_TMEM_FULL, abort_flag)) ok = false;
    __syncwarp();
    tc_fence_after();
    for (int c = 0; c < chunks; ++c) {
      uint32_t rg[HP];
      lt_tmem_load<HP>(tmem_O + lane_base + c * HP, rg);
      const int dim = c * 128 + key;
      if (dim < a.rank) {
        float* dst = a.scratch + first * a.ldc + dim;
        const int step = a.splits * a.ldc;
#pragma unroll
        for (int h = 0; h < HP; ++h, dst += step)
          if (h0 + h < a.H) *dst = __uint_as_float(rg[h]);
      }
      __syncwarp();
    }
    tc_fence_before();
  } else if (threadIdx.x < HP && h0 + threadIdx.x < a.H) {
    float* ml = a.scratch + (long long)a.B * a.n * a.H * a.splits * a.ldc + 2 * (((long long)r * a.H + h0 + threadIdx.x) * a.splits + split);
    ml[0] = -INFINITY;
    ml[1] = 0.f;
  }
  __syncthreads();
  if (*abort_flag) {
    for (int k = 0; k < 64; ++k) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 5) { tc_fence_after(); tmem_dealloc(tmem_S, cols); }
}

// Heads per CTA, 64-column panels of a row, tiles in flight and shared memory; false when a row is too long.
static bool lt_plan(const gb_ll_latent_args& a, int* hp, int* panels, int* stages, size_t* smem) {
  *panels = (a.rank + a.dr + 63) / 64;
  const int for_values = 2 * ((a.rank + 127) / 128);
  if (*panels < for_values) *panels = for_values;
  for (int h = a.H <= 16 ? 16 : 32; h >= 16; h -= 16)
    for (int s = 2; s >= 1; --s) {
      const size_t need = (size_t)s * *panels * AT_N * 128 + (size_t)(*panels + 2) * h * 128 + LT_BAR_BYTES + 1024;
      if (need > LT_SMEM_MAX - 2048 || h * (1 + (a.rank + 127) / 128) > 256) continue;
      *hp = h; *stages = s; *smem = need;
      return true;
    }
  return false;
}

template <int HP>
static int lt_go(const gb_ll_latent_args& a, int panels, int stages, size_t smem, cudaStream_t st) {
  CUtensorMap tc, tq;
  const uint64_t rows = (uint64_t)a.B * a.n;
  if (gb_make_tmap_2d_16b(&tc, a.cache, (uint64_t)a.B * a.cap, a.ldc, a.ldc, AT_N, 64, 1)) return -20;
  if (gb_make_tmap_2d_16b(&tq, a.qa16, rows * a.heads_pad, (uint64_t)panels * 64, (uint64_t)panels * 64, HP, 64, 1)) return -21;
  GB_PDL_LAUNCH_SMEM(ll_latent_tc_kernel<HP>, dim3((unsigned)(rows * (a.heads_pad / HP)), a.splits), dim3(LT_THREADS), smem, st, tc, tq, a, panels, stages);
  return gb_launch_rc();
}

}  // namespace gb

using namespace gb;

// 0 when the tensor-core kernel covers the shapes: then the padded head count and the row length of qa16.
extern "C" int gb_ll_latent_tc_plan(const gb_ll_latent_args* p, int* heads_pad, int* ld_qa16) {
  int hp, panels, stages;
  size_t smem;
  if (!p || !heads_pad || !ld_qa16 || p->dtype != 1 || p->cap % AT_N || (long long)p->B * p->cap > 0x7fffffffll || p->ldc % 8) return -1;
  if (!lt_plan(*p, &hp, &panels, &stages, &smem)) return -2;
  *heads_pad = (p->H + hp - 1) / hp * hp;
  *ld_qa16 = panels * 64;
  return 0;
}

// Partial results of `splits` runs of tiles into scratch (gb_ll_latent_attn goes on from there).
extern "C" int gb_ll_latent_tc(const gb_ll_latent_args* p, cudaStream_t st) {
  int hp, panels, stages, pad, ld;
  size_t smem;
  if (const int rc = gb_ll_latent_tc_plan(p, &pad, &ld)) return rc;
  if (!p->qa16 || !p->cache || !p->scratch || !p->st || !p->status || p->heads_pad != pad || p->ld_qa16 != ld || p->B <= 0 || p->n <= 0 || p->splits < 1) return -1;
  lt_plan(*p, &hp, &panels, &stages, &smem);
  return hp == 32 ? lt_go<32>(*p, panels, stages, smem, st) : lt_go<16>(*p, panels, stages, smem, st);
}
