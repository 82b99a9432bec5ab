// Kernels of models described layer by layer (attention with a kept-prefix window, sink, output gate, capped scores, distance
// bias; attention over a shared latent; Mamba-2; dense feed-forward; norms on the sublayers' outputs or ahead of them).  Every kernel works on `B` sequences of `n` consecutive new tokens
// (row r = b * n + t) that continue from the per-sequence state in `st` (position of the first new token: abs_pos),
// so a prompt, a portion of one and a single decoded token are the same call.  Sizes are run-time values; rows of
// weights and activations that feed a matrix product are padded with zeros to a multiple of eight elements.
//
// dtype: element type of weights, activations and attention cache: 1 = bf16, 2 = fp32.  What belongs to the state (SSM
// states, positions), norms, scores, gates of the recurrence and the residual is fp32 for either.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "gb_decode.h"

#ifdef __cplusplus
extern "C" {
#endif

// x[r, :] = table[ids[r], :] in fp32 (pitch d) and in the compute type (pitch ld16; the columns past d are zeroed).
int gb_ll_embed(const int* ids, const void* table, long long ld_table, int vocab, float* x, void* x16, long long ld16, int rows,
                int d, int dtype, cudaStream_t st);
// x_out = x + (y / rms(y)) * w, x16 = compute-type copy of x_out.  x16 may be NULL; x_out may be x.
int gb_ll_postnorm(const float* y, long long ldy, const float* x, const float* w, float eps, float* x_out, void* x16,
                   long long ld16, int rows, int d, int dtype, cudaStream_t st);
// out[r, :] = compute-type copy of (x / rms(x)) * w for x row `row_idx[r]` (NULL: row r).
int gb_ll_norm_rows(const float* x, const int* row_idx, const float* w, float eps, void* out, long long ldo, int rows, int d,
                    int dtype, cudaStream_t st);
// The norm of a model: mode 0, x / rms(x) * w; mode 1, (x - mean) / sqrt(variance + eps) * w + b.
#define GB_LL_NORM_RMS 0
#define GB_LL_NORM_LAYER 1
// x[r, :] = norm(table[ids[r], :]) in fp32 (pitch d).
int gb_ll_embed_norm(const int* ids, const void* table, long long ld_table, int vocab, int mode, const float* w, const float* b, float eps,
                     float* x, int rows, int d, int dtype, cudaStream_t st);
// v = x + alpha * y + x0 (y, x0 may be NULL); x_out = v unless NULL (may be x); out = compute-type copy of norm(v) unless NULL
// (columns past d zeroed).  Row r reads x row `row_idx[r]` when given (then without y, x0 and x_out).
int gb_ll_add_norm(const float* y, long long ldy, float alpha, const float* x, const float* x0, const int* row_idx, int mode,
                   const float* w, const float* b, float eps, float* x_out, void* out, long long ldo, int rows, int d, int dtype,
                   cudaStream_t st);
// v = max(v, 0)^2 in place over [rows, n] fp32.
int gb_ll_relu2_f32(float* v, long long ld, int rows, int n, cudaStream_t st);
// v = cap * tanh(v / cap) in place over [rows, n] fp32.
int gb_ll_softcap(float* v, long long ld, int rows, int n, float cap, cudaStream_t st);
// C[M, N] = A[M, K] B[N, K]^T in fp32 (true fp32 products); K a multiple of 4, rows 16-byte aligned.
int gb_ll_gemm_f32(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc, int M, int N, int K,
                   cudaStream_t st);
// act[r, j] = silu(g) * u for gate/up columns interleaved in blocks of 64 (g0..g63, u0..u63, g64..), fp32.
int gb_ll_swiglu_f32(const float* gu, long long ld, float* act, long long lda, int rows, int E, cudaStream_t st);
// st[b].abs_pos += n (and the cache_len the sampler's transcript shares), pos_out[b] = new position.
int gb_ll_advance(gb_seq_state* state, int* pos_out, int B, int n, cudaStream_t st);

// ------------------------------------------------------------------------------------------------ token-step GEMV
// out[b, j] = W[j, :] . v_b for B <= 8 sequences, where v_b is made by a prologue inside the kernel:
//   prologue 0: v = x16 (compute type, pitch ldx)
//   prologue 1: x_new = x + norm(y) * w1 (y NULL: x_new = x), written to x_out by one block; v = x_new, or
//               norm(x_new) * w2 when w2 is given
//   prologue 2: v = norm_parts(y16 * silu(z16)) * w1, `parts` equal parts each by its own root mean square
//   prologue 3: the same from v32 = y silu(z) (fp32, pitch d) and `n_sq` sums of squares per sequence, n_sq / parts to a part
//   prologue 4: v = x16 / rms(x16) * w1 (x16 fully read by every block)
//   prologue 5: x_new = x + alpha * y + x0 (y, x0 may be NULL), written to x_out by one block; v = norm(x_new) with w1, b1
//               and norm_mode (GB_LL_NORM_*)
// n1 > 0: rows from n1 on go to out2 (compute type, pitch ldo2) as max(v, 0)^2.
// swiglu != 0: W holds gate/up rows interleaved in blocks of 64 (N = 2 E rows) and out[b, j] = silu(gate_j) * up_j.
// softcap > 0: out = cap * tanh(out / cap).
typedef struct gb_ll_gemv_args {
  const void* W; int fmt, N, K;          // K: stored row length (values beyond `d` are zero)
  int B, dtype, prologue, swiglu;
  int d;                                 // true length of v
  const void* x16; long long ldx;
  const float* x; const float* y; long long ldy; const float* w1; const float* w2; float eps; float* x_out;
  const void* y16; long long ldy16; const void* z16; long long ldz; int parts;
  const float* v32; const float* sq; int n_sq;
  void* out; long long ldo; int out_f32; float softcap;
  const float* x0; float alpha; const float* b1; int norm_mode;
  int n1; void* out2; long long ldo2;
} gb_ll_gemv_args;
int gb_ll_gemv(const gb_ll_gemv_args* a, cudaStream_t st);

// ------------------------------------------------------------------------------------------------ attention
// Cache rows of a sequence: positions below `keep` have row = position for good; later positions share a ring,
// row = keep + (position - keep) % (cap - keep).  Key j is visible to query i iff j <= i and (window == 0 or
// i - j < window or j < keep).  The ring must hold window - 1 + n positions (all of them when window == 0).
typedef struct gb_ll_attn_args {
  int dtype, B, n;
  int H, G;                              // query heads, key/value heads
  int dk, dv, dkp, dvp;                  // head sizes and their padded row lengths in q and the caches (padding is zero)
  int rot_dims, rot_half;                // rotated leading dimensions; 0: pairs (2i, 2i+1), 1: pairs (i, i + rot_dims/2)
  const double* freq;                    // [rot_dims / 2] angular frequencies
  const float* cs;                       // optional [rows, rot_dims / 2, 2]: cosines and sines of this call's rows
                                         // (gb_ll_rotations); NULL: computed on the spot
  int qk_norm;                           // divide q and k by their root mean square after the rotation
  float eps, scale;
  int window, keep, cap;
  const void* proj; long long ld_proj;   // [rows, q: H*dk | k: G*dk | v: G*dv ..]
  const void* gate; long long ld_gate;   // [rows, H*dv] or NULL: the heads' outputs are multiplied by its sigmoid
  const float* sink;                     // [H] or NULL: exp(sink) joins the soft-max denominator
  float softcap;                         // > 0: score = softcap * tanh(score / softcap)
  const float* slopes;                   // [H] or NULL: score -= slope * (i - j), after the cap
  float temp_coef; int temp_every;       // temp_every > 0: q *= 1 + temp_coef * ln(floor((i + 1) / temp_every) + 1)
  void* q;                               // [rows, H, dkp]
  void* cache_k; void* cache_v;          // [B, cap, ld_k]: head g at column g*dkp / [B, cap, ld_v]: at g*dvp
  long long ld_k, ld_v;
  void* out; long long ldo;              // [rows, H*dv]
  float* scratch; int splits;            // token step: B * H * splits * (dvp + 2) floats: partial outputs,
                                         // then (maximum, sum) pairs
  const gb_seq_state* st;
  int pos0_max;                          // host's upper bound of abs_pos over the B sequences (tile counts); -1 unknown
  int* status;
} gb_ll_attn_args;
// gb_ll_qkv_store writes caches with ld_k = G*dkp and ld_v = G*dvp.
int gb_ll_rotations(const double* freq, int pairs, const gb_seq_state* st, int B, int n, float* cs, cudaStream_t stream);
int gb_ll_qkv_store(const gb_ll_attn_args* a, cudaStream_t st);     // rotation, norm, q out, k and v into the cache
int gb_ll_attn_prefill(const gb_ll_attn_args* a, cudaStream_t st);  // any dtype and head size up to 256
int gb_ll_attn_tc_ok(const gb_ll_attn_args* a);                     // 0 when the tensor-core kernel covers the shapes
int gb_ll_attn_tc(const gb_ll_attn_args* a, cudaStream_t st);       // bf16
int gb_ll_attn_decode(const gb_ll_attn_args* a, cudaStream_t st);   // n == 1

// ------------------------------------------------------------------------------------------------ attention over a latent
// What a position leaves in the cache is one row [c: rank | k_rot: dr | zeros up to ldc]: the normed latent, from which each
// head's unrotated key and value are linear maps, and the rotated key part that all heads share.
//   Many new tokens: keys and values of every position so far are made by one product with W_kv (whose rows carry k_rot
//   into every head's key) and the kernels above run on them.
//   Few new tokens: the query goes through its head's key map instead (gb_ll_latent_absorb), all heads attend to the cache
//   rows themselves (value = the first `rank` numbers of the key), and the value map follows the soft-max
//   (gb_ll_latent_attn).
typedef struct gb_ll_latent_args {
  int dtype, B, n;                       // B sequences of n new tokens, rows r = b * n + t
  int H, dn, dr, dv, rank, q_rank;       // heads, unrotated / rotated query-key size, value size, latent sizes
  int dkp, dvp, rot_dims;                // padded head sizes; rotated leading dimensions of the dr (interleaved pairs)
  const float* cs;                       // [rows, rot_dims / 2, 2] (gb_ll_rotations)
  float eps, scale;
  const void* proj; long long ld_proj;   // [rows, query latent: q_rank | latent: rank | k_rot: dr | gate: H*dv ..]
  const float* q_norm; const float* kv_norm;
  void* cq; long long ld_cq;             // [rows, q_rank] normed query latent (columns past q_rank zeroed)
  void* cache; int ldc; int cap;         // [B, cap, ldc]
  const void* qc; long long ld_qc;       // [rows, H, dn + dr] queries as projected
  void* q;                               // [rows, H, dkp] rotated queries
  const void* W_kv; long long ld_w;      // rows h*dkp + d: key map of head h, rows H*dkp + h*dvp + e: its value map; columns: rank ..
  float* qa;                             // [rows, H, ldc] queries against cache rows, or
  void* qa16; int heads_pad, ld_qa16;    // [rows, heads_pad, ld_qa16] the same in bf16 for the tensor cores (padding is zero)
  const void* gate; long long ld_gate;   // [rows, H*dv] or NULL
  void* out; long long ldo;              // [rows, H*dv]
  float* scratch; int splits;            // rows * H * splits * (ldc + 2) floats: partial outputs [.., ldc], then (maximum, sum)
  const gb_seq_state* st; int* status;
} gb_ll_latent_args;
int gb_ll_latent_store(const gb_ll_latent_args* a, cudaStream_t st);    // norms, rotation of k_rot: cq and the cache rows
int gb_ll_latent_queries(const gb_ll_latent_args* a, cudaStream_t st);  // q = qc with its rotated part turned, padded
int gb_ll_latent_absorb(const gb_ll_latent_args* a, int store, cudaStream_t st);   // qa or qa16; store != 0: the cache rows, too
int gb_ll_latent_attn(const gb_ll_latent_args* a, cudaStream_t st);     // rank + dr up to 1024; on the tensor cores with qa16
// 0 when the tensor-core kernel covers the shapes (bf16, cap a multiple of 128): heads_pad and ld_qa16 to use.
int gb_ll_latent_tc_plan(const gb_ll_latent_args* a, int* heads_pad, int* ld_qa16);
int gb_ll_latent_tc(const gb_ll_latent_args* a, cudaStream_t st);       // the part of gb_ll_latent_attn before the merge

// ------------------------------------------------------------------------------------------------ Mamba-2
typedef struct gb_ll_mamba_args {
  int dtype, B, n;
  int H, P, N, G, taps;                  // heads, head size, state size, groups, convolution taps
  int Pp, Np;                            // padded row lengths of xh and bc / cc
  int Ns;                                // row length of a stored state (N rounded up to 4)
  const void* proj; long long ld_proj;   // [rows, z: H*P | x: H*P | B: G*N | C: G*N | dt: H]
  const float* conv_w; const float* conv_b;   // [channels, taps], [channels] for channels x | B | C
  const float* dt_bias; const float* A_log; const float* D;
  const float* norm_w; int norm_groups; float eps;
  void* conv_state;                      // [B, taps, channels]: input of position p in row p % taps
  float* ssm;                            // [B, H, P, Ns]
  void* xh; void* bc; void* cc;          // convolved: [rows, H, Pp], [rows, G, Np], [rows, G, Np]
  void* y; long long ld_y;               // [rows, H*P]
  void* out; long long ld_out;           // [rows, H*P] gated and normed
  float* gated; float* gated_sq;         // token step, optional: y silu(z) [B, H*P] and its sums of squares [B, H, ceil(P/32)]
                                         // instead of y
  const gb_seq_state* st;
  float* chunk_ws;                       // chunked scan: gb_ll_ssd_ws_floats floats, or NULL (no cutting into segments)
  int* status;
} gb_ll_mamba_args;
int gb_ll_conv(const gb_ll_mamba_args* a, cudaStream_t st);
int gb_ll_scan(const gb_ll_mamba_args* a, cudaStream_t st);         // recurrence token by token, any dtype
// The recurrence in chunks of 128 tokens on the tensor cores: bf16, P <= 128, N <= 128, Pp 64 or 128, Np 128.  `segments`:
// runs that a sequence is cut into, 0 = by the number of SMs.
int gb_ll_ssd_ok(const gb_ll_mamba_args* a);                        // 0 when the shapes are covered
long long gb_ll_ssd_ws_floats(int B, int H, int P, int Ns, int n, int segments);
int gb_ll_ssd(const gb_ll_mamba_args* a, int segments, cudaStream_t st);
int gb_ll_gated_norm(const gb_ll_mamba_args* a, cudaStream_t st);
int gb_ll_mamba_step(const gb_ll_mamba_args* a, cudaStream_t st);   // n == 1: convolution + recurrence in one kernel

#ifdef __cplusplus
}
#endif
