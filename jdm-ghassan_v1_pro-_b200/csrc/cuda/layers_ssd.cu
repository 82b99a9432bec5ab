// Mamba-2 state recurrence over many tokens on the tensor cores (interface in gb_layers.h): chunks of 128 tokens, the
// state of a head resident in tensor memory from chunk to chunk.
//
// With L_t the running sum of the log decays inside a chunk (fp32), the chunk's outputs and its new state are
//   y_t = sum_{s <= t} (C_t . B_s) exp(L_t - L_s) dt_s x_s  +  exp(L_t) C_t . S_prev  +  D x_t
//   S   = exp(L_last) S_prev + sum_s exp(L_last - L_s) dt_s B_s x_s^T
// (the block form of the recurrence: T. Dao, A. Gu, "Transformers are SSMs", 2024).  x, B and C are bf16 as the
// convolution leaves them.  Everything else is fp32; where an fp32 quantity has to be an operand (the weights of the
// first sum, the scaled x of the state update, S_prev itself) it enters as two bf16 terms, value and remainder, so that
// products keep 16 bits of it, and the state accumulates in fp32.
//
// One CTA per (sequence, head, run of chunks): warps 0-7 own the chunk's token rows (weights of the first sum, outputs;
// warps w and w + 4 share 32 rows and take alternate 32-column blocks), warps 8-11 the state rows and the scaled x, warp 12
// loads tiles with TMA, warp 13 issues the MMAs, warp 14 turns raw step sizes into dt and L one chunk ahead.  The state
// chain (S_prev -> operand, scaled x, state update) runs ahead of the output chain.  When there are fewer heads than SMs
// the tokens are cut into segments: a first launch computes what every segment adds to the state from zero, a small
// kernel turns those into the state before each segment, the last launch starts from there.
#include <algorithm>

#include "sm100_common.cuh"
#include "gb_layers.h"
#include "tc_tiles.cuh"
#include "layers_util.cuh"

namespace gb {

constexpr int SD_Q = 128;                  // tokens per chunk
constexpr int SD_N = 128;                  // padded state size

struct SsdParams {
  int B, n, H, P, N, G, Ns;
  const __nv_bfloat16* proj; long long ld_proj; int dt_col;
  const float* dt_bias; const float* A_log; const float* D;
  float* ssm;
  __nv_bfloat16* y; long long ld_y;
  const gb_seq_state* st;
  int n_chunks, seg_chunks, n_seg;
  float* ws_state;                         // [B, H, n_seg, P, Ns]: slot k = state before segment k (first launch: slot 0 as it
                                           // is, slot k + 1 = what segment k adds from zero)
  float* ws_decay;                         // [B, H, n_seg]: log2 decay over segment k
  int* status;
};

__device__ __forceinline__ float sd_ex2(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

// MMA and commit for a warp that runs converged: every lane passes the same operands, the lane with `on` != 0 issues.  The
// operands then stay in uniform registers, which is where the instruction wants them; issued from a one-lane branch, each
// MMA first moved its descriptors there and cost 70 to 100 cycles of issue time.
__device__ __forceinline__ void sd_mma(uint32_t on, uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      :
      : "r"(d), "l"(a), "l"(b), "r"(idesc), "r"(accumulate), "r"(on)
      : "memory");
}
__device__ __forceinline__ void sd_mma_ts(uint32_t on, uint32_t d, uint32_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "setp.ne.b32 q, %5, 0;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      :
      : "r"(d), "r"(a), "l"(b), "r"(idesc), "r"(accumulate), "r"(on)
      : "memory");
}
__device__ __forceinline__ void sd_commit(uint32_t on, uint64_t* bar) {
  asm volatile(
      "{\n\t.reg .pred q;\n\t"
      "setp.ne.b32 q, %1, 0;\n\t"
      "@q tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}"
      :
      : "r"(smem_u32(bar)), "r"(on)
      : "memory");
}

// Out of line: the kernel has five roles with long straight-line bodies, and what bounds it once the chains overlap is the
// instruction cache (a wait that was over cost 400 cycles with everything unrolled and inlined).
__device__ __noinline__ bool sd_wait(uint32_t bar, uint32_t parity, int* status, int code, volatile int* abort_flag) {
  const long long t0 = clock64();
  for (;;) {
#pragma unroll 1
    for (int i = 0; i < 1024; ++i) {
      uint32_t ok;
      asm volatile(
          "{\n\t.reg .pred P1;\n\t"
          "mbarrier.try_wait.parity.shared::cta.b64 P1, [%1], %2;\n\t"
          "selp.b32 %0, 1, 0, P1;\n\t}"
          : "=r"(ok)
          : "r"(bar), "r"(parity)
          : "memory");
      if (ok) return true;
    }
    if (*abort_flag) return false;
    if (clock64() - t0 > 4000000000LL) {
      atomicCAS(status, 0, code);
      *abort_flag = 1;
      return false;
    }
  }
}

// 2 values -> packed bf16 pair and the packed remainders
__device__ __forceinline__ void sd_split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = Cvt<__nv_bfloat16>::pack2(a, b);
  const float2 h = Cvt<__nv_bfloat16>::unpack2(hi);
  lo = Cvt<__nv_bfloat16>::pack2(a - h.x, b - h.y);
}

// SO: the state-only pass, without the token-row warps, C, and the state as an operand: two CTAs share an SM (head size 64).
template <int PP, bool SO>
struct SsdCfg {
  static constexpr int W_STATE = SO ? 0 : 8, W_TMA = W_STATE + 4, W_MMA = W_STATE + 5, W_DT = W_STATE + 6;
  static constexpr int THREADS = (W_DT + 1) * 32, CTAS = SO && PP == 64 ? 2 : 1;
  static constexpr int STAGES = !SO && PP == 64 ? 2 : 1;
  static constexpr int NG = PP == 64 ? 2 : 1;                       // score buffers in tensor memory
  static constexpr uint32_t TBC = SD_Q * SD_N * 2, TX = SD_Q * PP * 2;
  static constexpr uint32_t OFF_B = SO ? 0 : TBC, OFF_X = OFF_B + TBC, STAGE = OFF_X + TX;      // a stage: C, B, x
  static constexpr uint32_t TS = SO ? 0 : SD_N * PP * 2;
  static constexpr size_t TILES = (size_t)STAGES * STAGE + 2 * TS + 2 * TX;
  static constexpr size_t SMEM = TILES + 2 * (2 * SD_Q + 96) * 4 + 128;
  // the products with both terms of S_prev side by side (one pass over C) where tensor memory has the columns
  static constexpr int NY2 = PP == 64 ? 2 : 1;
  static constexpr int COL_Y = 128 * NG, COL_Y2 = COL_Y + PP, COL_S = SO ? 0 : COL_Y2 + PP * NY2;
  static constexpr int COLS = SO ? PP : 512;
};

template <int PP, bool SO>
__global__ void __launch_bounds__(SsdCfg<PP, SO>::THREADS, SsdCfg<PP, SO>::CTAS) ll_ssd_kernel(const __grid_constant__ CUtensorMap tmX,
                                                               const __grid_constant__ CUtensorMap tmB,
                                                               const __grid_constant__ CUtensorMap tmC,
                                                               const __grid_constant__ SsdParams p) {
  using T = __nv_bfloat16;
  using K = SsdCfg<PP, SO>;
  extern __shared__ __align__(1024) uint8_t smem[];
  if (smem_u32(smem) & 1023u) {            // no static shared memory: the dynamic window starts aligned
    if (threadIdx.x == 0) atomicCAS(p.status, 0, ST_BAD_ARGUMENT);
    return;
  }
  uint8_t* sShi = smem + K::STAGES * K::STAGE;
  uint8_t* sSlo = sShi + K::TS;
  uint8_t* sXhi = sSlo + K::TS;
  uint8_t* sXlo = sXhi + K::TX;
  float* sL = reinterpret_cast<float*>(sXlo + K::TX);       // [2][128] L in log2 units
  float* sV = sL + 2 * SD_Q;                                // [2][128] log2(dt) - L
  float* sU = sV + 2 * SD_Q;                                // [2][96] dt exp(L_end - L), L_end = L at the end of the token's 32-block
  uint64_t* bars = reinterpret_cast<uint64_t*>(sU + 2 * 96);
  uint64_t* full = bars;               // 2
  uint64_t* empty = bars + 2;          // 2
  uint64_t* l_full = bars + 4;         // 2
  uint64_t* l_empty = bars + 6;        // 2
  uint64_t* g_full = bars + 8;
  uint64_t* m_ready = bars + 9;
  uint64_t* y_full = bars + 10;
  uint64_t* y_empty = bars + 11;
  uint64_t* s_ready = bars + 12;
  uint64_t* xw_ready = bars + 13;
  uint64_t* s_full = bars + 14;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr bool so = SO;
  const int seg = blockIdx.x % (so ? p.n_seg - 1 : p.n_seg), bh = blockIdx.x / (so ? p.n_seg - 1 : p.n_seg);
  const int b = bh / p.H, h = bh - b * p.H, g = h / (p.H / p.G);
  const int c_lo = seg * p.seg_chunks, c_hi = min(p.n_chunks, c_lo + p.seg_chunks), nc = c_hi - c_lo;

  if (threadIdx.x == 0) {
    for (int s = 0; s < 2; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], so ? 1 : 9);
      mbar_init(&l_full[s], 1);
      mbar_init(&l_empty[s], so ? 4 : 12);
    }
    mbar_init(g_full, 1);
    mbar_init(m_ready, 8);
    mbar_init(y_full, 1);
    mbar_init(y_empty, 8);
    mbar_init(s_ready, 4);
    mbar_init(xw_ready, 4);
    mbar_init(s_full, 1);
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == K::W_MMA) { tmem_alloc(tmem_slot, K::COLS); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // with all 512 columns the allocation starts at column 0 (checked), and the addresses below are constants
  const uint32_t tm = so ? *tmem_slot : 0u;
  if (!so && *tmem_slot != 0 && threadIdx.x == 0) { atomicCAS(p.status, 0, ST_BAD_ARGUMENT); *abort_flag = 1; }
  const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
#define SD_WAIT(bar, ph, code) if (!sd_wait(smem_u32(bar), ph, p.status, code, abort_flag)) break

  if (warp == K::W_TMA) {
    // ------------------------------------------------------------------ TMA
    if (lane == 0) {
      for (int c = 0; c < nc; ++c) {
        const int s = c % K::STAGES, ph = (c / K::STAGES) & 1;
        SD_WAIT(&empty[s], ph ^ 1, ST_TIMEOUT_EMPTY);
        uint8_t* st = smem + s * K::STAGE;
        const int row = b * p.n + (c_lo + c) * SD_Q;
        mbar_arrive_expect_tx(&full[s], K::STAGE);
        load_tile<SD_N>(&tmB, &full[s], st + K::OFF_B, g * SD_N, row);
        load_tile<PP>(&tmX, &full[s], st + K::OFF_X, h * PP, row);
        if (!so) load_tile<SD_N>(&tmC, &full[s], st, g * SD_N, row);
      }
    }
    __syncwarp();
  } else if (warp == K::W_MMA) {
    // ------------------------------------------------------------------ MMA
    {
      const uint32_t on = lane == 0;
      const uint32_t id_g = make_idesc_f16(1, 0, 0, SD_Q, SD_Q);
      const uint32_t id_y = make_idesc_f16(1, 0, 1, SD_Q, PP);
      const uint32_t id_y2 = make_idesc_f16(1, 0, 1, SD_Q, PP * K::NY2);
      const uint32_t id_s = make_idesc_f16(1, 1, 1, SD_N, PP);
      // Descriptors advance by address alone (units of 16 bytes): a tile of 128 rows has panels of 1024 units, a step of 16
      // along K is 2 units inside a K-major panel and 128 units (16 rows) in an MN-major one.
      const uint64_t d_st = make_smem_desc_sw128(smem_u32(smem), 16, 1024), d_mn = make_smem_desc_sw128(smem_u32(smem), SD_Q * 128, 1024);
      const uint64_t d_s = make_smem_desc_sw128(smem_u32(sShi), SD_N * 128, 1024), d_xw = make_smem_desc_sw128(smem_u32(sXhi), SD_Q * 128, 1024);
      auto scores = [&](int c) {
        const uint64_t dc = d_st + (c % K::STAGES) * (K::STAGE >> 4);
        const uint32_t to = (c % K::NG) * 128;
#pragma unroll
        for (int kk = 0; kk < SD_N / 16; ++kk) {
          const uint32_t off = (kk >> 2) * 1024 + (kk & 3) * 2;
          sd_mma(on, to, dc + off, dc + (K::OFF_B >> 4) + off, id_g, kk ? 1u : 0u);
        }
        sd_commit(on, g_full);
      };
      bool ok = true;
      if (!so) {
        ok = sd_wait(smem_u32(&full[0]), 0, p.status, ST_TIMEOUT_FULL, abort_flag);
        if (ok) { tc_fence_after(); scores(0); }
      }
      for (int c = 0; c < nc && ok; ++c) {
        const int s = c % K::STAGES;
        const uint64_t dc = d_st + s * (K::STAGE >> 4), dmn = d_mn + s * (K::STAGE >> 4);
        if (so) SD_WAIT(&full[s], (c / K::STAGES) & 1, ST_TIMEOUT_FULL);
        SD_WAIT(s_ready, c & 1, ST_TIMEOUT_EMPTY);
        if (!so) {
          if (c > 0) SD_WAIT(y_empty, (c - 1) & 1, ST_TIMEOUT_TMEM_EMPTY);
          tc_fence_after();
#pragma unroll
          for (int part = 0; part < 2 / K::NY2; ++part)
#pragma unroll
            for (int kk = 0; kk < SD_N / 16; ++kk)
              sd_mma(on, K::COL_Y2, dc + (kk >> 2) * 1024 + (kk & 3) * 2, d_s + part * (K::TS >> 4) + kk * 128, id_y2, (part || kk) ? 1u : 0u);
        }
        SD_WAIT(xw_ready, c & 1, ST_TIMEOUT_EMPTY);
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int kk = 0; kk < SD_Q / 16; ++kk)
            sd_mma(on, tm + K::COL_S, dmn + (K::OFF_B >> 4) + kk * 128, d_xw + part * (K::TX >> 4) + kk * 128, id_s, 1u);
        sd_commit(on, s_full);
        if (!so) {
          SD_WAIT(m_ready, c & 1, ST_TIMEOUT_TMEM_EMPTY);
          tc_fence_after();
          const uint32_t m0 = (c % K::NG) * 128;
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int kk = 0; kk < SD_Q / 16; ++kk)
              sd_mma_ts(on, K::COL_Y, m0 + (kk >> 1) * 32 + part * 16 + (kk & 1) * 8, dmn + (K::OFF_X >> 4) + kk * 128, id_y,
                          (part || kk) ? 1u : 0u);
          sd_commit(on, y_full);
        }
        sd_commit(on, &empty[s]);
        if (!so && c + 1 < nc) {
          if (K::NG == 1) SD_WAIT(y_full, c & 1, ST_TIMEOUT_TMEM_FULL);      // the one score buffer still holds this chunk's weights
          SD_WAIT(&full[(c + 1) % K::STAGES], ((c + 1) / K::STAGES) & 1, ST_TIMEOUT_FULL);
          tc_fence_after();
          scores(c + 1);
        }
      }
    }
    __syncwarp();
  } else if (warp == K::W_DT) {
    // ------------------------------------------------------------------ dt and L
    const float bias = p.dt_bias[h], na2 = -expf(p.A_log[h]) * 1.4426950408889634f;
    for (int c = 0; c < nc; ++c) {
      const int s = c & 1, t0 = (c_lo + c) * SD_Q + lane * 4;
      float dt[4], cum[4], run = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        dt[k] = t0 + k < p.n ? ll_softplus(Cvt<T>::to_f(p.proj[((long long)b * p.n + t0 + k) * p.ld_proj + p.dt_col + h]) + bias) : 0.f;
        run += na2 * dt[k];
        cum[k] = run;
      }
      float inc = run;                                     // inclusive sum over lanes
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= o) inc += v;
      }
      const float before = inc - run;
      // L at the end of this lane's 32-token block
      const float Lb = __shfl_sync(0xffffffffu, before + cum[3], lane | 7);
      SD_WAIT(&l_empty[s], ((c >> 1) & 1) ^ 1, ST_TIMEOUT_EMPTY);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float L = before + cum[k];
        sL[s * SD_Q + lane * 4 + k] = L;
        sV[s * SD_Q + lane * 4 + k] = log2f(dt[k]) - L;
        if (lane < 24) sU[s * 96 + lane * 4 + k] = dt[k] * sd_ex2(Lb - L);
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&l_full[s]);
    }
    __syncwarp();
  } else if (warp < K::W_STATE) {
    // ------------------------------------------------------------------ token rows
    const int quarter = warp & 3, half = warp >> 2, r = quarter * 32 + lane;
    const float D = p.D[h];
    for (int c = 0; c < nc && !so; ++c) {
      const int ls = c & 1, s = c % K::STAGES, t = (c_lo + c) * SD_Q + r;
      SD_WAIT(&l_full[ls], (c >> 1) & 1, ST_TIMEOUT_FULL);
      const float* Lrow = sL + ls * SD_Q;
      const float L = Lrow[r];
      const uint32_t tg = tm + (c % K::NG) * 128 + lane_base;
      SD_WAIT(g_full, c & 1, ST_TIMEOUT_TMEM_FULL);
      tc_fence_after();
      // weights (C_t . B_s) exp(L_t - L_s) dt_s, written over the scores they come from: per 32 columns, 16 columns of
      // packed values and 16 of packed remainders.  Left of the diagonal block the exponential is a product of a factor
      // of the row and one of the column, both against the L at the end of the column's block (neither exceeds 1).
#pragma unroll 1
      for (int q = half; q < 4; q += 2) {
        uint32_t hi[16], lo[16];
        if (q < quarter) {
          uint32_t rg[32];
          tmem_ld_32x32(tg + q * 32, rg);
          const float f = sd_ex2(L - Lrow[q * 32 + 31]);
          const float4* u4 = reinterpret_cast<const float4*>(sU + ls * 96) + q * 8;
          tmem_ld_wait();
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const float4 u = u4[k];
            sd_split2(__uint_as_float(rg[4 * k]) * (f * u.x), __uint_as_float(rg[4 * k + 1]) * (f * u.y), hi[2 * k], lo[2 * k]);
            sd_split2(__uint_as_float(rg[4 * k + 2]) * (f * u.z), __uint_as_float(rg[4 * k + 3]) * (f * u.w), hi[2 * k + 1], lo[2 * k + 1]);
          }
        } else if (q == quarter) {
          uint32_t rg[32];
          tmem_ld_32x32(tg + q * 32, rg);
          const float4* v4 = reinterpret_cast<const float4*>(sV + ls * SD_Q) + q * 8;
          tmem_ld_wait();
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const float4 v = v4[k];
            float m[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) m[e] = 4 * k + e > lane ? 0.f : __uint_as_float(rg[4 * k + e]) * sd_ex2(L + m[e]);
            sd_split2(m[0], m[1], hi[2 * k], lo[2 * k]);
            sd_split2(m[2], m[3], hi[2 * k + 1], lo[2 * k + 1]);
          }
          __syncwarp();
        } else {
#pragma unroll
          for (int k = 0; k < 16; ++k) { hi[k] = 0u; lo[k] = 0u; }
        }
        tmem_st_32x16(tg + q * 32, hi);
        tmem_st_32x16(tg + q * 32 + 16, lo);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(m_ready);
      const float eL = sd_ex2(L);
      const uint8_t* sx = smem + s * K::STAGE + K::OFF_X;
      T* yp = p.y + ((long long)b * p.n + t) * p.ld_y + h * p.P;
      const bool live = t < p.n;
      const bool vec = p.P == PP && ((reinterpret_cast<uintptr_t>(p.y) | (uintptr_t)(p.ld_y * 2)) & 15) == 0;
      SD_WAIT(y_full, c & 1, ST_TIMEOUT_TMEM_FULL);
      SD_WAIT(&full[s], (c / K::STAGES) & 1, ST_TIMEOUT_FULL);      // long since true; this thread reads x itself
      tc_fence_after();
#pragma unroll 1
      for (int c0 = half * (PP / 2); c0 < (half + 1) * (PP / 2); c0 += 16) {
        uint32_t a[16], e[16];
        tmem_ld_32x16(tm + K::COL_Y + lane_base + c0, a);
        tmem_ld_32x16(tm + K::COL_Y2 + lane_base + c0, e);
        if constexpr (K::NY2 == 2) {
          uint32_t e2[16];
          tmem_ld_32x16(tm + K::COL_Y2 + PP + lane_base + c0, e2);
          tmem_ld_wait();
#pragma unroll
          for (int k = 0; k < 16; ++k) e[k] = __float_as_uint(__uint_as_float(e[k]) + __uint_as_float(e2[k]));
        } else {
          tmem_ld_wait();
        }
#pragma unroll
        for (int k = 0; k < 2 && live; ++k) {
          const int col = c0 + 8 * k;
          const uint4 xq = *reinterpret_cast<const uint4*>(sx + (col >> 6) * (SD_Q * 128) + sw128_off(r, col & 63));
          const uint32_t xw[4] = {xq.x, xq.y, xq.z, xq.w};
          float v[8];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float2 x = Cvt<T>::unpack2(xw[j]);
            v[2 * j] = __uint_as_float(a[8 * k + 2 * j]) + eL * __uint_as_float(e[8 * k + 2 * j]) + D * x.x;
            v[2 * j + 1] = __uint_as_float(a[8 * k + 2 * j + 1]) + eL * __uint_as_float(e[8 * k + 2 * j + 1]) + D * x.y;
          }
          if (vec) {
            uint4 o;
            o.x = Cvt<T>::pack2(v[0], v[1]); o.y = Cvt<T>::pack2(v[2], v[3]);
            o.z = Cvt<T>::pack2(v[4], v[5]); o.w = Cvt<T>::pack2(v[6], v[7]);
            *reinterpret_cast<uint4*>(yp + col) = o;
          } else {
#pragma unroll
            for (int j = 0; j < 8; ++j)
              if (col + j < p.P) yp[col + j] = Cvt<T>::from_f(v[j]);
          }
        }
        __syncwarp();                       // the next tensor-memory access is the whole warp's
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) { mbar_arrive(y_empty); mbar_arrive(&empty[s]); mbar_arrive(&l_empty[ls]); }
    }
  } else {
    // ------------------------------------------------------------------ state rows and scaled x
    const int r = threadIdx.x - K::W_STATE * 32;   // state column (0 .. 127) / token of the chunk
    const bool live_n = r < p.N;
    const long long per = (long long)p.P * p.Ns;
    float* home = p.ssm + bh * per;
    float* ws = p.ws_state ? p.ws_state + (long long)bh * p.n_seg * per : nullptr;
    const uint32_t ts = tm + K::COL_S + lane_base;
    const bool fresh = p.st[b].abs_pos == 0;
    // the state this run starts from
    const float* from = so || (p.n_seg == 1 && fresh) ? nullptr : p.n_seg == 1 ? home : ws + seg * per;
#pragma unroll
    for (int q = 0; q < PP / 16; ++q) {
      uint32_t v[16];
#pragma unroll
      for (int k = 0; k < 16; ++k) {
        const int pp = q * 16 + k;
        v[k] = (from && live_n && pp < p.P) ? __float_as_uint(from[(long long)pp * p.Ns + r]) : 0u;
      }
      __syncwarp();
      tmem_st_32x16(ts + q * 16, v);
    }
    tmem_st_wait();
    if (so && seg == 0 && live_n)                       // the last launch's last segment replaces `home`
      for (int pp = 0; pp < p.P; ++pp) ws[(long long)pp * p.Ns + r] = fresh ? 0.f : home[(long long)pp * p.Ns + r];
    float total = 0.f;
    bool ok = true;
    for (int c = 0; c < nc; ++c) {
      const int ls = c & 1, s = c % K::STAGES;
      ok = false;
      SD_WAIT(&l_full[ls], (c >> 1) & 1, ST_TIMEOUT_FULL);
      const float Ll = sL[ls * SD_Q + SD_Q - 1], dec = sd_ex2(Ll), w = sd_ex2(Ll + sV[ls * SD_Q + r]);
      total += Ll;
      if (c > 0) SD_WAIT(s_full, (c - 1) & 1, ST_TIMEOUT_TMEM_FULL);
      tc_fence_after();
#pragma unroll 1
      for (int q = 0; q < PP / 32; ++q) {
        uint32_t v[32];
        tmem_ld_32x32(ts + q * 32, v);
        tmem_ld_wait();
        if (!so) {
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            uint4 hi, lo;
            sd_split2(__uint_as_float(v[8 * k]), __uint_as_float(v[8 * k + 1]), hi.x, lo.x);
            sd_split2(__uint_as_float(v[8 * k + 2]), __uint_as_float(v[8 * k + 3]), hi.y, lo.y);
            sd_split2(__uint_as_float(v[8 * k + 4]), __uint_as_float(v[8 * k + 5]), hi.z, lo.z);
            sd_split2(__uint_as_float(v[8 * k + 6]), __uint_as_float(v[8 * k + 7]), hi.w, lo.w);
            const int col = q * 32 + 8 * k;
            const uint32_t off = (col >> 6) * (SD_N * 128) + sw128_off(r, col & 63);
            *reinterpret_cast<uint4*>(sShi + off) = hi;
            *reinterpret_cast<uint4*>(sSlo + off) = lo;
          }
        }
        uint32_t w0[16], w1[16];
#pragma unroll
        for (int k = 0; k < 16; ++k) {
          w0[k] = __float_as_uint(__uint_as_float(v[k]) * dec);
          w1[k] = __float_as_uint(__uint_as_float(v[16 + k]) * dec);
        }
        tmem_st_32x16(ts + q * 32, w0);
        tmem_st_32x16(ts + q * 32 + 16, w1);
      }
      tmem_st_wait();
      tc_fence_before();
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(s_ready);
      SD_WAIT(&full[s], (c / K::STAGES) & 1, ST_TIMEOUT_FULL);
      const uint8_t* sx = smem + s * K::STAGE + K::OFF_X;
#pragma unroll 4
      for (int q = 0; q < PP / 8; ++q) {
        const uint32_t off = (q >> 3) * (SD_Q * 128) + sw128_off(r, (q & 7) * 8);
        const uint4 xq = *reinterpret_cast<const uint4*>(sx + off);
        const uint32_t xw[4] = {xq.x, xq.y, xq.z, xq.w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 x = Cvt<T>::unpack2(xw[j]);
          sd_split2(x.x * w, x.y * w, hi[j], lo[j]);
        }
        *reinterpret_cast<uint4*>(sXhi + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(sXlo + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) { mbar_arrive(xw_ready); mbar_arrive(&l_empty[ls]); }
      ok = true;
    }
    if (ok && nc > 0 && sd_wait(smem_u32(s_full), (nc - 1) & 1, p.status, ST_TIMEOUT_TMEM_FULL, abort_flag)) {
      tc_fence_after();
      float* dst = so ? ws + (seg + 1) * per : (seg == p.n_seg - 1 ? home : nullptr);
#pragma unroll 1
      for (int q = 0; q < PP / 16; ++q) {
        uint32_t v[16];
        tmem_ld_32x16(ts + q * 16, v);
        tmem_ld_wait();
        if (dst && live_n) {
#pragma unroll
          for (int k = 0; k < 16; ++k)
            if (q * 16 + k < p.P) dst[(long long)(q * 16 + k) * p.Ns + r] = __uint_as_float(v[k]);
        }
        __syncwarp();
      }
      if (so && r == 0) p.ws_decay[(long long)bh * p.n_seg + seg] = total;
      tc_fence_before();
    }
  }
#undef SD_WAIT
  __syncthreads();
  if (*abort_flag) {
    for (int k = 0; k < 64; ++k) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == K::W_MMA) { tc_fence_after(); tmem_dealloc(*tmem_slot, K::COLS); }
}

// ws slots 1 .. n_seg - 1 from "what segment k adds" to "state before the segment"; one thread per state value.
__global__ void __launch_bounds__(256) ll_ssd_combine_kernel(float* __restrict__ ws, const float* __restrict__ decay, int n_seg, long long per) {
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= per) return;
  float* w = ws + (long long)blockIdx.y * n_seg * per + i;
  const float* d = decay + (long long)blockIdx.y * n_seg;
  float s = w[0];
#pragma unroll 4
  for (int k = 1; k < n_seg; ++k) {
    s = s * sd_ex2(d[k - 1]) + w[k * per];
    w[k * per] = s;
  }
}

struct SsdPlan { int n_chunks, seg_chunks, n_seg; };

// Segments per head: the cheapest number of rounds over the SMs.  A CTA costs about three chunks to start and drain; a
// state-only chunk about 0.7 of a full one, and two state-only CTAs share an SM.
static SsdPlan ssd_plan(int BH, int n, int sms) {
  SsdPlan best{(n + SD_Q - 1) / SD_Q, 0, 1};
  best.seg_chunks = best.n_chunks;
  double cost = (double)((BH + sms - 1) / sms) * (best.n_chunks + 3.0);
  for (int s = 2; s <= 16 && s <= best.n_chunks; ++s) {
    const int per = (best.n_chunks + s - 1) / s, k = (best.n_chunks + per - 1) / per;
    const double c = (per + 3.0) * ((BH * k + sms - 1) / sms) + (0.7 * per + 3.0) * ((BH * (k - 1) + 2 * sms - 1) / (2 * sms)) + 3.0;
    if (c < cost * 0.95) { cost = c; best.seg_chunks = per; best.n_seg = k; }
  }
  return best;
}

static int ssd_sms() {
  static int sms = 0;
  if (!sms) {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) sms = 0;
  }
  return sms;
}

template <int PP, bool SO>
static int ssd_attr() {
  static bool done = false;
  if (!done) {
    if (cudaFuncSetAttribute(ll_ssd_kernel<PP, SO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SsdCfg<PP, SO>::SMEM) != cudaSuccess) return -10;
    if (SO) (void)cudaFuncSetAttribute(ll_ssd_kernel<PP, SO>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    done = true;
  }
  return 0;
}

template <int PP>
static int ssd_go(const gb_ll_mamba_args& a, int force_segments, cudaStream_t st) {
  using K = SsdCfg<PP, false>;
  using KS = SsdCfg<PP, true>;
  static_assert(K::SMEM <= 232448 && K::COL_S + PP <= 512 && KS::CTAS * (KS::SMEM + 1024) <= 233472, "shared memory / tensor memory budget");
  const int sms = ssd_sms();
  if (sms <= 0 || ssd_attr<PP, false>() || ssd_attr<PP, true>()) return -10;
  CUtensorMap tx, tb, tc;
  const uint64_t rows = (uint64_t)a.B * a.n;
  if (gb_make_tmap_2d_16b(&tx, a.xh, rows, (uint64_t)a.H * PP, (uint64_t)a.H * PP, SD_Q, 64, 1)) return -20;
  if (gb_make_tmap_2d_16b(&tb, a.bc, rows, (uint64_t)a.G * SD_N, (uint64_t)a.G * SD_N, SD_Q, 64, 1)) return -21;
  if (gb_make_tmap_2d_16b(&tc, a.cc, rows, (uint64_t)a.G * SD_N, (uint64_t)a.G * SD_N, SD_Q, 64, 1)) return -22;
  SsdPlan plan = ssd_plan(a.B * a.H, a.n, sms);
  if (force_segments > 0) {
    const int per = (plan.n_chunks + force_segments - 1) / force_segments;
    plan.seg_chunks = per;
    plan.n_seg = (plan.n_chunks + per - 1) / per;
  }
  if (!a.chunk_ws) { plan.n_seg = 1; plan.seg_chunks = plan.n_chunks; }
  SsdParams p{};
  p.B = a.B; p.n = a.n; p.H = a.H; p.P = a.P; p.N = a.N; p.G = a.G; p.Ns = a.Ns;
  p.proj = static_cast<const __nv_bfloat16*>(a.proj); p.ld_proj = a.ld_proj; p.dt_col = 2 * a.H * a.P + 2 * a.G * a.N;
  p.dt_bias = a.dt_bias; p.A_log = a.A_log; p.D = a.D; p.ssm = a.ssm;
  p.y = static_cast<__nv_bfloat16*>(a.y); p.ld_y = a.ld_y; p.st = a.st; p.status = a.status;
  p.n_chunks = plan.n_chunks; p.seg_chunks = plan.seg_chunks; p.n_seg = plan.n_seg;
  const long long BH = (long long)a.B * a.H;
  if (plan.n_seg > 1) {
    p.ws_state = a.chunk_ws;
    p.ws_decay = a.chunk_ws + BH * plan.n_seg * a.P * a.Ns;
    ll_ssd_kernel<PP, true><<<(unsigned)(BH * (plan.n_seg - 1)), KS::THREADS, KS::SMEM, st>>>(tx, tb, tc, p);
    const long long per = (long long)a.P * a.Ns;
    ll_ssd_combine_kernel<<<dim3((unsigned)((per + 255) / 256), (unsigned)BH), 256, 0, st>>>(p.ws_state, p.ws_decay, plan.n_seg, per);
  }
  ll_ssd_kernel<PP, false><<<(unsigned)(BH * plan.n_seg), K::THREADS, K::SMEM, st>>>(tx, tb, tc, p);
  return gb_launch_rc();
}

}  // namespace gb

using namespace gb;

extern "C" int gb_ll_ssd_ok(const gb_ll_mamba_args* p) {
  if (!p || p->dtype != 1) return -1;
  if ((p->Pp != 64 && p->Pp != 128) || p->Np != SD_N || p->P > p->Pp || p->N > p->Np) return -2;
  if ((long long)p->B * p->n > 0x7fffffffll) return -3;
  return 0;
}

extern "C" long long gb_ll_ssd_ws_floats(int B, int H, int P, int Ns, int n, int segments) {
  int k = segments;
  if (k <= 0) {
    const int sms = ssd_sms();
    k = ssd_plan(B * H, n, sms > 0 ? sms : 148).n_seg;
  }
  return k > 1 ? (long long)B * H * k * ((long long)P * Ns + 1) : 0;
}

extern "C" int gb_ll_ssd(const gb_ll_mamba_args* p, int segments, cudaStream_t st) {
  if (const int rc = gb_ll_ssd_ok(p)) return rc;
  if (!p->st || !p->proj || !p->xh || !p->bc || !p->cc || !p->y || !p->ssm || !p->status || !p->dt_bias || !p->A_log || !p->D ||
      p->B <= 0 || p->n <= 0 || p->G <= 0 || p->H % p->G || p->Ns < p->N) return -1;
  return p->Pp == 64 ? ssd_go<64>(*p, segments, st) : ssd_go<128>(*p, segments, st);
}
