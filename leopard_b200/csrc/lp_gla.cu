// leopard_b200 — linear attention with a data-dependent decay per KEY CHANNEL: a matrix memory per head whose rows fade at their own,
// token by token computed rates; everything after the projections in 32-bit floats.
//
// Per head, with q (scaled by q_scale), k [dim], v [vdim] and a decay pre-activation z [dim] of the token:
//   a = exp(-exp(z))  (LP_GLA_DECAY_DOUBLE_EXP)   or   a = sigmoid(z)^decay_exp  (LP_GLA_DECAY_SIGMOID_POW)
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T                                       S [dim, vdim], starts at zero
//   o_t = S_t^T q_t                             or, with a bonus u [dim]: o_t = (S_(t-1) + diag(u) k_t v_t^T)^T q_t
// then o / rms(o) per head (eps), times a gain per channel, times silu(g).
//
//   lp_gla     prompts, portions and one-token steps alike.  The recurrence runs in REGISTERS: a CTA per (piece of a request, head, tile of
//              32, 64 or 128 state columns), a warp owns 16 rows of the tile, a lane 1, 2 or 4 of its columns; two rows share an
//              instruction (packed fp32 multiply-adds).  Tokens are staged in shared memory 8 at a time, the next stage copied asynchronously
//              while one computes; the state updates of a stage need no synchronisation, the warps' partial read-outs meet in shared memory once
//              per stage, and there a warp per token closes the head: norm, gain, gate.
//     one piece per request   (one-token steps, short portions, batches that fill the GPU): the state comes from the request's slot and
//              goes back there.
//     pieces of a long prompt   three launches: (1) every piece but a request's last runs from a zero state and leaves its
//              contribution and the product of its decays, (2) a scan over a request's pieces turns those into the state at each
//              piece's start, (3) every piece runs from its start state and writes its outputs; the last one writes the slot.
//              Products of decays are used as they are (at most 1), so no logarithm is taken and nothing overflows.
//   A row's result is the token-by-token recurrence in every case, up to the grouping of the sums at a piece's start.
//   Value heads wider than 128 columns take several column tiles; their outputs go through a buffer and lp_gla's finish kernel.
#include <cuda_pipeline.h>
#include "lp_host.h"
#include "../../include/leopard_b200.h"

namespace lp {

typedef __nv_bfloat16 bf16;

constexpr int GLA_ROWS = 16;            // state rows per warp
constexpr int GLA_MAX_WARPS = 16;       // dim <= 256
constexpr int GLA_FUSED_COLS = 128;     // widest value head one CTA closes by itself

struct GlaArgs {
  const float* q; const float* k; const float* v; long long ldq, ldk, ldv;
  int heads, dim, vdim; float q_scale;
  int decay; float decay_exp;
  const float* z; long long ldz;
  const float* t; long long ldt; const bf16* w2; long long ldw2; int rank, t_tanh; const float* z_bias;
  const float* bonus;
  const float* out_gain; long long gain_stride; const float* gate; long long ldg; float eps;
  float* state; long long slot_stride;
  void* out; long long ldo; int out_fp32;
};

struct GlaBatch {
  const int *seq_row0, *seq_pos0, *seq_slot;
  const int *seq_chunk0, *chunk_seq, *chunk_row0, *chunk_len;      // pieces of `group` consecutive chunks; group 0: one piece per request
  int group;
  float* u;      // [chunk][head][dim][vdim]: a piece's contribution, then the state at its start (at the piece's first chunk)
  float* p;      // [chunk][head][dim]: the product of a piece's decays
  float* raw;    // [row][head][vdim]: outputs before the norm, when a head takes several column tiles
};

__device__ __forceinline__ float gla_decay(int kind, float e, float z) {
  if (kind == LP_GLA_DECAY_DOUBLE_EXP) return expf(-expf(z));
  // sigmoid(z)^e = exp(-e softplus(-z)); an absolute error of the logarithm is a relative one of the decay, so log(1 + x) serves
  return expf(-e * (logf(1.0f + expf(-fabsf(z))) + fmaxf(-z, 0.f)));
}

// the pre-activation of decay n of a row from the row's low-rank vector (t: activated when `active`)
__device__ __forceinline__ float gla_low_rank(const GlaArgs& a, const float* t, bool active, int n) {
  float z = a.z_bias != nullptr ? a.z_bias[n] : 0.f;
  const bf16* w = a.w2 + (long long)n * a.ldw2;
  int i = 0;
  if (active && ((reinterpret_cast<uintptr_t>(w) & 15) == 0)) {      // eight factors a read
    for (; i + 8 <= a.rank; i += 8) {
      const uint4 u = *reinterpret_cast<const uint4*>(w + i);
      const unsigned f[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        z = fmaf(__uint_as_float(f[j] << 16), t[i + 2 * j], z);
        z = fmaf(__uint_as_float(f[j] & 0xffff0000u), t[i + 2 * j + 1], z);
      }
    }
  }
  for (; i < a.rank; ++i) z = fmaf(__bfloat162float(w[i]), active || !a.t_tanh ? t[i] : tanhf(t[i]), z);
  return z;
}

__device__ __forceinline__ float gla_close(float o, float rinv, float gain, const float* gate) {
  float v = o * rinv * gain;
  if (gate != nullptr) v *= __fdividef(*gate, 1.0f + expf(-*gate));
  return v;
}
__device__ __forceinline__ void gla_store(const GlaArgs& a, long long row, int h, int c, float v) {
  const long long at = row * a.ldo + h * a.vdim + c;
  if (a.out_fp32) reinterpret_cast<float*>(a.out)[at] = v;
  else reinterpret_cast<bf16*>(a.out)[at] = __float2bfloat16(v);
}

constexpr int GLA_TOK = 8;              // tokens a stage

// One operand of a stage: `n` floats of each of nt tokens (src_ld apart) into rows of dst, by all threads of the CTA; a thread's place (token
// t, column c) in the stage is the caller's, `t_step` tokens further on each turn.
__device__ __forceinline__ void gla_fetch(float* dst, int dst_ld, const float* src, long long src_ld, int n, int nt, int t, int c, int t_step,
                                          bool vec) {
  if (c >= n) return;
  for (; t < nt; t += t_step) {
    const float* from = src + t * src_ld + c;
    float* to = dst + t * dst_ld + c;
    if (vec) {
      __pipeline_memcpy_async(to, from, 16);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (c + i < n) __pipeline_memcpy_async(to + i, from + i, 4);
    }
  }
}

// OUT: read-outs, from the stored state (group 0: the request's slot; else the piece's start state in u).  !OUT: contribution and decay
// product of the pieces that another piece follows.  The operands of a stage are copied asynchronously while the stage before computes.
template <int CPL, bool OUT, bool BONUS>
__global__ void __launch_bounds__(GLA_MAX_WARPS * 32)
gla_run_kernel(GlaArgs a, GlaBatch b, int vec) {
  extern __shared__ float dyn_smem[];
  constexpr int COLS = 32 * CPL, TOK = GLA_TOK;
  const int h = blockIdx.y, col0 = blockIdx.z * COLS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, NW = blockDim.x >> 5, dpad = NW * GLA_ROWS;
  int s, row0, len;
  bool last = true;
  if (b.group == 0) {
    s = blockIdx.x;
    row0 = b.seq_row0[s];
    len = b.seq_row0[s + 1] - row0;
  } else {
    const int c = blockIdx.x;
    s = b.chunk_seq[c];
    const int c_end = b.seq_chunk0[s + 1];
    if ((c - b.seq_chunk0[s]) % b.group != 0) return;
    const int c_last = (c + b.group < c_end ? c + b.group : c_end) - 1;
    last = c_last == c_end - 1;
    if (!OUT && last) return;
    row0 = b.chunk_row0[c];
    len = b.chunk_row0[c_last] + b.chunk_len[c_last] - row0;
  }
  // two stages of [k | z, turned into decays | v | (OUT) q | (OUT) gate], zero beyond dim and vdim
  const int part = TOK * dpad, stage = (OUT ? 3 : 2) * part + (OUT ? 2 : 1) * TOK * COLS;
  float* red_s = dyn_smem + 2 * stage;          // OUT: [TOK][NW][COLS] partial read-outs; else [2][dpad] partial decay products
  float* bon_s = red_s + TOK * NW * COLS;       // OUT: [TOK] sum_d bonus_d q_d k_d
  const int cols = a.vdim - col0 < COLS ? a.vdim - col0 : COLS;
  const bool gated = OUT && a.gate != nullptr && b.raw == nullptr;
  if (a.dim < dpad || cols < COLS)
    for (int i = tid; i < 2 * stage; i += blockDim.x) dyn_smem[i] = 0.f;
  if (a.dim < dpad || cols < COLS) __syncthreads();
  // four columns a thread: the 2 dpad threads cover 8 tokens of dpad channels at once, and a tile's columns in 32 NW / (COLS / 4) tokens a turn
  const int f_t = tid / (dpad >> 2), f_c = tid % (dpad >> 2) * 4;
  const int v_t = tid / (COLS / 4), v_c = tid % (COLS / 4) * 4, v_step = NW * 32 / (COLS / 4);
  auto fetch = [&](int t0, int buf) {
    const int nt = len - t0 < TOK ? len - t0 : TOK;
    float* p = dyn_smem + buf * stage;
    const long long row = row0 + t0;
    gla_fetch(p, dpad, a.k + row * a.ldk + h * a.dim, a.ldk, a.dim, nt, f_t, f_c, TOK, vec);
    if (a.z != nullptr) gla_fetch(p + part, dpad, a.z + row * a.ldz + h * a.dim, a.ldz, a.dim, nt, f_t, f_c, TOK, vec);
    p += 2 * part;
    gla_fetch(p, COLS, a.v + row * a.ldv + h * a.vdim + col0, a.ldv, cols, nt, v_t, v_c, v_step, vec);
    p += TOK * COLS;
    if (OUT) gla_fetch(p, dpad, a.q + row * a.ldq + h * a.dim, a.ldq, a.dim, nt, f_t, f_c, TOK, vec);
    if (gated) gla_fetch(p + part, COLS, a.gate + row * a.ldg + h * a.vdim + col0, a.ldg, cols, nt, v_t, v_c, v_step, vec);
    __pipeline_commit();
  };
  fetch(0, 0);
  const long long hs = (long long)a.dim * a.vdim;
  float* slot = a.state + (long long)b.seq_slot[s] * a.slot_stride + h * hs;
  float* piece = b.group ? b.u + ((long long)blockIdx.x * a.heads + h) * hs : nullptr;
  const float* src = b.group ? piece : slot;
  const bool stored = OUT && (b.group ? true : b.seq_pos0[s] > 0);
  // S[rr][c]: rows 2 rr, 2 rr + 1 of the warp's 16, column lane + 32 c
  float2 S[GLA_ROWS / 2][CPL];
#pragma unroll
  for (int rr = 0; rr < GLA_ROWS / 2; ++rr)
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      const int d = warp * GLA_ROWS + 2 * rr, y = col0 + lane + 32 * c;
      S[rr][c].x = (stored && d < a.dim && y < a.vdim) ? src[(long long)d * a.vdim + y] : 0.f;
      S[rr][c].y = (stored && d + 1 < a.dim && y < a.vdim) ? src[(long long)(d + 1) * a.vdim + y] : 0.f;
    }
  // without z the decays come from the low-rank vectors; a lone token's is activated once, ahead of its use
  const bool low = a.z == nullptr, lone = low && len == 1 && OUT && a.rank <= TOK * NW * COLS;
  if (lone)
    for (int i = tid; i < a.rank; i += blockDim.x) {
      const float t = a.t[row0 * a.ldt + i];
      red_s[i] = a.t_tanh ? tanhf(t) : t;
    }
  // a thread turns one channel's pre-activations into decays, every other token's (the CTA has two threads per channel)
  const int my_d = tid % dpad, my_t = tid / dpad;
  float prod = 1.f;
  float gain[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const int y = lane + 32 * c;
    gain[c] = OUT && a.out_gain != nullptr && b.raw == nullptr && y < a.vdim ? a.out_gain[h * a.gain_stride + y] : 1.0f;
  }
  for (int t0 = 0, buf = 0; t0 < len; t0 += TOK, buf ^= 1) {
    const int nt = len - t0 < TOK ? len - t0 : TOK;
    __pipeline_wait_prior(0);
    __syncthreads();      // this stage has arrived, the one before has been read
    if (t0 + TOK < len) fetch(t0 + TOK, buf ^ 1);
    const float* k_s = dyn_smem + buf * stage;
    float* w_s = dyn_smem + buf * stage + part;
    const float* v_s = w_s + part;
    const float* q_s = v_s + TOK * COLS;
    const float* g_s = q_s + part;
    if (my_d < a.dim) {
#pragma unroll
      for (int j = 0; j < TOK / 2; ++j) {
        const int t = my_t + 2 * j;
        if (t < nt) {
          float z;
          if (!low) z = w_s[t * dpad + my_d];
          else z = gla_low_rank(a, lone ? red_s : a.t + (row0 + t0 + t) * a.ldt, lone, h * a.dim + my_d);
          const float w = gla_decay(a.decay, a.decay_exp, z);
          w_s[t * dpad + my_d] = w;
          if (!OUT) prod *= w;
        }
      }
    }
    if (BONUS) {      // a warp per token; read after the next barrier but one
      for (int t = warp; t < nt; t += NW) {
        float acc = 0.f;
        for (int d = lane; d < a.dim; d += 32) acc = fmaf(a.bonus[h * a.dim + d] * q_s[t * dpad + d], k_s[t * dpad + d], acc);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (lane == 0) bon_s[t] = acc;
      }
    }
    __syncthreads();
#pragma unroll(CPL == 4 ? 2 : 1)
    for (int t = 0; t < nt; ++t) {
      float2 vv[CPL], acc[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        const float x = v_s[t * COLS + lane + 32 * c];
        vv[c] = make_float2(x, x);
        acc[c] = make_float2(0.f, 0.f);
      }
      const float4* k4 = reinterpret_cast<const float4*>(k_s + t * dpad + warp * GLA_ROWS);
      const float4* w4 = reinterpret_cast<const float4*>(w_s + t * dpad + warp * GLA_ROWS);
      const float4* q4 = reinterpret_cast<const float4*>(q_s + t * dpad + warp * GLA_ROWS);
#pragma unroll
      for (int r4 = 0; r4 < GLA_ROWS / 4; ++r4) {
        const float4 kk = k4[r4], ww = w4[r4];
        float4 qq;
        if (OUT) qq = q4[r4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const float2 k2 = half ? make_float2(kk.z, kk.w) : make_float2(kk.x, kk.y);
          const float2 w2 = half ? make_float2(ww.z, ww.w) : make_float2(ww.x, ww.y);
          float2 q2;
          if (OUT) q2 = half ? make_float2(qq.z, qq.w) : make_float2(qq.x, qq.y);
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            float2& st = S[2 * r4 + half][c];
            if (OUT && BONUS) acc[c] = fma2(st, q2, acc[c]);      // the state before this token
            st = fma2(w2, st, mul2(k2, vv[c]));
            if (OUT && !BONUS) acc[c] = fma2(st, q2, acc[c]);
          }
        }
      }
      if (OUT) {
#pragma unroll
        for (int c = 0; c < CPL; ++c) red_s[(t * NW + warp) * COLS + lane + 32 * c] = acc[c].x + acc[c].y;
      }
    }
    if (OUT) {
      __syncthreads();
      for (int t = warp; t < nt; t += NW) {      // a warp closes a token
        const long long row = row0 + t0 + t;
        float o[CPL], ss = 0.f;
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          float x = BONUS ? bon_s[t] * v_s[t * COLS + lane + 32 * c] : 0.f;
#pragma unroll 4
          for (int y = 0; y < NW; ++y) x += red_s[(t * NW + y) * COLS + lane + 32 * c];
          o[c] = x * a.q_scale;
          ss = fmaf(o[c], o[c], ss);      // columns past vdim are zero
        }
        if (b.raw != nullptr) {
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            const int y = col0 + lane + 32 * c;
            if (y < a.vdim) b.raw[(row * a.heads + h) * a.vdim + y] = o[c];
          }
          continue;
        }
#pragma unroll
        for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
        const float rinv = 1.0f / sqrtf(ss / (float)a.vdim + a.eps);
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          const int y = lane + 32 * c;
          if (y < a.vdim) gla_store(a, row, h, y, gla_close(o[c], rinv, gain[c], gated ? g_s + t * COLS + y : nullptr));
        }
      }
    }
  }
  if (!OUT) {      // the product of the piece's decays: two partial products per channel
    red_s[my_t * dpad + my_d] = prod;
    __syncthreads();
    if (blockIdx.z == 0 && my_t == 0 && my_d < a.dim)
      b.p[((long long)blockIdx.x * a.heads + h) * a.dim + my_d] = red_s[my_d] * red_s[dpad + my_d];
  }
  if (!OUT || last) {
    float* dst = OUT ? slot : piece;
#pragma unroll
    for (int rr = 0; rr < GLA_ROWS / 2; ++rr)
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        const int d = warp * GLA_ROWS + 2 * rr, y = col0 + lane + 32 * c;
        if (d < a.dim && y < a.vdim) dst[(long long)d * a.vdim + y] = S[rr][c].x;
        if (d + 1 < a.dim && y < a.vdim) dst[(long long)(d + 1) * a.vdim + y] = S[rr][c].y;
      }
  }
}

// one thread per state element of a (request, head): u[piece] <- state at the piece's start.  The pieces' contributions are loaded
// several at a time (independent loads) ahead of the dependent multiply-adds.
constexpr int GLA_SCAN_THREADS = 256, GLA_SCAN_BATCH = 16;
__global__ void __launch_bounds__(GLA_SCAN_THREADS)
gla_scan_kernel(GlaArgs a, GlaBatch b) {
  const int s = blockIdx.x, h = blockIdx.y;
  const long long hs = (long long)a.dim * a.vdim;
  const long long i = (long long)blockIdx.z * GLA_SCAN_THREADS + threadIdx.x;
  if (i >= hs) return;
  const int d = (int)(i / a.vdim);
  const int c0 = b.seq_chunk0[s], c1 = b.seq_chunk0[s + 1];
  const int n = (c1 - c0 + b.group - 1) / b.group;      // pieces; the last one's contribution is not needed
  float S = b.seq_pos0[s] > 0 ? a.state[(long long)b.seq_slot[s] * a.slot_stride + h * hs + i] : 0.f;
  float* u = b.u + ((long long)c0 * a.heads + h) * hs + i;
  const float* p = b.p + ((long long)c0 * a.heads + h) * a.dim + d;
  const long long us = (long long)b.group * a.heads * hs, ps = (long long)b.group * a.heads * a.dim;
  for (int j = 0; j < n; j += GLA_SCAN_BATCH) {
    float own[GLA_SCAN_BATCH], dec[GLA_SCAN_BATCH];
#pragma unroll
    for (int k = 0; k < GLA_SCAN_BATCH; ++k) {
      const bool live = j + k < n - 1;
      own[k] = live ? u[k * us] : 0.f;
      dec[k] = live ? p[k * ps] : 1.f;
    }
#pragma unroll
    for (int k = 0; k < GLA_SCAN_BATCH; ++k) {
      if (j + k < n) {
        u[k * us] = S;
        S = fmaf(dec[k], S, own[k]);
      }
    }
    u += GLA_SCAN_BATCH * us;
    p += GLA_SCAN_BATCH * ps;
  }
}

constexpr int GLA_FIN_WARPS = 4;
__global__ void __launch_bounds__(GLA_FIN_WARPS * 32)
gla_finish_kernel(GlaArgs a, int R, const float* __restrict__ raw) {
  const int item = blockIdx.x * GLA_FIN_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= R * a.heads) return;
  const int row = item / a.heads, h = item % a.heads;
  const float* o = raw + (long long)item * a.vdim;
  float ss = 0.f;
  for (int c = lane; c < a.vdim; c += 32) ss = fmaf(o[c], o[c], ss);
#pragma unroll
  for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  const float rinv = 1.0f / sqrtf(ss / (float)a.vdim + a.eps);
  for (int c = lane; c < a.vdim; c += 32) 
    gla_store(a, row, h, c, gla_close(o[c], rinv, a.out_gain != nullptr ? a.out_gain[h * a.gain_stride + c] : 1.0f,
                                      a.gate != nullptr ? a.gate + (long long)row * a.ldg + h * a.vdim + c : nullptr));
}

// the operand of the low-rank decay product: act(t) as fp32, or split into two bf16 values hi + lo side by side (a product with the
// weight written twice then loses 16 bits less than one with a rounded operand)
__global__ void lowrank_operand_kernel(const float* __restrict__ t, long long ldt, int R, int rank, int act_tanh, float* __restrict__ out_f32,
                                       bf16* __restrict__ out_split, long long ldo) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)R * rank) return;
  const long long m = i / rank, c = i % rank;
  float v = t[m * ldt + c];
  if (act_tanh) v = tanhf(v);
  if (out_f32 != nullptr) {
    out_f32[m * ldo + c] = v;
  } else {
    const bf16 hi = __float2bfloat16(v);
    out_split[m * ldo + c] = hi;
    out_split[m * ldo + rank + c] = __float2bfloat16(v - __bfloat162float(hi));
  }
}

template <int CPL>
static size_t gla_smem_bytes(int warps, bool out) {
  constexpr int COLS = 32 * CPL;
  const size_t dpad = (size_t)warps * GLA_ROWS;
  const size_t stage = (out ? 3 : 2) * GLA_TOK * dpad + (out ? 2 : 1) * GLA_TOK * COLS;
  return (2 * stage + (out ? (size_t)GLA_TOK * warps * COLS + GLA_TOK : 2 * dpad)) * sizeof(float);
}

template <int CPL, bool OUT, bool BONUS>
static int launch_gla_run(const GlaArgs& a, const GlaBatch& b, int pieces, int vec, cudaStream_t stream) {
  const int warps = (a.dim + GLA_ROWS - 1) / GLA_ROWS;
  const size_t smem = gla_smem_bytes<CPL>(warps, OUT);
  static size_t have = 48 * 1024;      // raised once per instantiation, and only for head sizes that need it
  if (smem > have) {
    LP_CHECK_CUDA(cudaFuncSetAttribute(gla_run_kernel<CPL, OUT, BONUS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    have = 160 * 1024;
  }
  const dim3 grid(pieces, a.heads, (a.vdim + 32 * CPL - 1) / (32 * CPL));
  gla_run_kernel<CPL, OUT, BONUS><<<grid, warps * 32, smem, stream>>>(a, b, vec);
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

template <int CPL>
static int launch_gla_out(const GlaArgs& a, const GlaBatch& b, int pieces, int vec, cudaStream_t stream) {
  if (a.bonus != nullptr) return launch_gla_run<CPL, true, true>(a, b, pieces, vec, stream);
  return launch_gla_run<CPL, true, false>(a, b, pieces, vec, stream);
}

template <int CPL>
static int launch_gla(const GlaArgs& a, GlaBatch b, int n_seqs, int n_chunks, int vec, cudaStream_t stream) {
  if (b.group == 0) {
    note_launch();
    return launch_gla_out<CPL>(a, b, n_seqs, vec, stream);
  }
  if (int rc = launch_gla_run<CPL, false, false>(a, b, n_chunks, vec, stream)) return rc;
  const long long hs = (long long)a.dim * a.vdim;
  gla_scan_kernel<<<dim3(n_seqs, a.heads, (unsigned)((hs + GLA_SCAN_THREADS - 1) / GLA_SCAN_THREADS)), GLA_SCAN_THREADS, 0, stream>>>(a, b);
  LP_CHECK_CUDA(cudaGetLastError());
  note_launch(3);
  return launch_gla_out<CPL>(a, b, n_chunks, vec, stream);
}

// 16-byte copies need every operand's base and row stride, and the heads inside a row, on 16-byte boundaries
static bool gla_vec(const GlaArgs& a) {
  const void* bases[] = {a.q, a.k, a.v, a.z, a.gate};
  for (const void* p : bases)
    if (p != nullptr && (reinterpret_cast<uintptr_t>(p) & 15)) return false;
  return a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ldq % 4 == 0 && a.ldk % 4 == 0 && a.ldv % 4 == 0 && (a.z == nullptr || a.ldz % 4 == 0) &&
         (a.gate == nullptr || a.ldg % 4 == 0);
}

static int gla_col_tiles(int vdim) { return (vdim + GLA_FUSED_COLS - 1) / GLA_FUSED_COLS; }

// chunks per piece, 0: one piece per request.  Long requests are cut when whole requests would leave multiprocessors idle (or wait for
// one long request); pieces are as long as still gives every multiprocessor several CTAs.
constexpr int GLA_CTAS_PER_SM = 8;
static int gla_group(int n_seqs, int n_chunks, int R, int longest, int heads, int tiles) {
  if (longest <= 2 * LP_RETENTION_CHUNK) return 0;
  const long long whole = (long long)n_seqs * heads * tiles;
  if (whole >= 4LL * sm_count() && (long long)longest * n_seqs <= 2LL * R) return 0;
  const long long g = (long long)n_chunks * heads * tiles / ((long long)sm_count() * GLA_CTAS_PER_SM);
  return (int)(g < 1 ? 1 : g > 16 ? 16 : g);
}

}  // namespace lp

using namespace lp;

extern "C" size_t lp_gla_workspace_bytes(int n_chunks, int R, int longest, int heads, int dim, int vdim) {
  size_t floats = vdim > GLA_FUSED_COLS ? (size_t)R * heads * vdim : 0;
  if (longest > 2 * LP_RETENTION_CHUNK) floats += (size_t)n_chunks * heads * ((size_t)dim * vdim + dim);
  return floats * sizeof(float);
}

extern "C" int lp_gla(const lp_gla_desc* d, int n_seqs, int n_chunks, int R, int longest, const int* seq_row0, const int* seq_pos0,
                      const int* seq_slot, const int* seq_chunk0, const int* chunk_seq, const int* chunk_row0, const int* chunk_len,
                      void* ws, size_t ws_bytes, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(d != nullptr && d->q != nullptr && d->k != nullptr && d->v != nullptr && d->state != nullptr && d->out != nullptr,
             "lp_gla: null operand");
  LP_REQUIRE(d->heads > 0 && d->dim > 0 && d->vdim > 0 && d->dim <= GLA_MAX_WARPS * GLA_ROWS, "lp_gla: bad sizes heads=%d dim=%d (at most %d) vdim=%d",
             d->heads, d->dim, GLA_MAX_WARPS * GLA_ROWS, d->vdim);
  LP_REQUIRE(d->decay == LP_GLA_DECAY_DOUBLE_EXP || d->decay == LP_GLA_DECAY_SIGMOID_POW, "lp_gla: unknown decay %d", d->decay);
  LP_REQUIRE(d->z != nullptr || (d->t != nullptr && d->w2 != nullptr && d->rank > 0), "lp_gla: neither decays nor their low-rank factors");
  LP_REQUIRE(d->slot_stride >= (long long)d->heads * d->dim * d->vdim, "lp_gla: a slot is smaller than the state");
  LP_REQUIRE(seq_row0 != nullptr && seq_pos0 != nullptr && seq_slot != nullptr && n_seqs >= 0 && R >= 0 && longest >= 0, "lp_gla: bad batch tables");
  if (n_seqs == 0 || R == 0) return 0;
  GlaArgs a;
  a.q = d->q; a.k = d->k; a.v = d->v; a.ldq = d->ldq; a.ldk = d->ldk; a.ldv = d->ldv; a.heads = d->heads; a.dim = d->dim; a.vdim = d->vdim;
  a.q_scale = d->q_scale; a.decay = d->decay; a.decay_exp = d->decay_exp; a.z = d->z; a.ldz = d->ldz; a.t = d->t; a.ldt = d->ldt;
  a.w2 = reinterpret_cast<const bf16*>(d->w2); a.ldw2 = d->ldw2; a.rank = d->rank; a.t_tanh = d->t_tanh; a.z_bias = d->z_bias;
  a.bonus = d->bonus; a.out_gain = d->out_gain; a.gain_stride = d->gain_stride; a.gate = d->gate; a.ldg = d->ldg; a.eps = d->eps;
  a.state = d->state; a.slot_stride = d->slot_stride; a.out = d->out; a.ldo = d->ldo; a.out_fp32 = d->out_fp32;
  GlaBatch b;
  b.seq_row0 = seq_row0; b.seq_pos0 = seq_pos0; b.seq_slot = seq_slot; b.seq_chunk0 = seq_chunk0; b.chunk_seq = chunk_seq;
  b.chunk_row0 = chunk_row0; b.chunk_len = chunk_len;
  b.group = gla_group(n_seqs, n_chunks, R, longest, d->heads, gla_col_tiles(d->vdim));
  LP_REQUIRE(b.group == 0 || (n_chunks > 0 && seq_chunk0 != nullptr && chunk_seq != nullptr && chunk_row0 != nullptr && chunk_len != nullptr),
             "lp_gla: null operand");
  const size_t need = lp_gla_workspace_bytes(n_chunks, R, longest, d->heads, d->dim, d->vdim);
  LP_REQUIRE(need == 0 || (ws != nullptr && ws_bytes >= need), "lp_gla: workspace too small");
  float* f = reinterpret_cast<float*>(ws);
  b.raw = d->vdim > GLA_FUSED_COLS ? f : nullptr;
  if (b.raw != nullptr) f += (size_t)R * d->heads * d->vdim;
  b.u = f;
  b.p = b.group ? f + (size_t)n_chunks * d->heads * d->dim * d->vdim : nullptr;
  const int vec = gla_vec(a) ? 1 : 0;
  int rc;
  if (d->vdim <= 32) rc = launch_gla<1>(a, b, n_seqs, n_chunks, vec, stream);
  else if (d->vdim <= 64) rc = launch_gla<2>(a, b, n_seqs, n_chunks, vec, stream);
  else rc = launch_gla<4>(a, b, n_seqs, n_chunks, vec, stream);
  if (rc != 0) return rc;
  if (b.raw != nullptr) {
    gla_finish_kernel<<<(R * d->heads + GLA_FIN_WARPS - 1) / GLA_FIN_WARPS, GLA_FIN_WARPS * 32, 0, stream>>>(a, R, b.raw);
    LP_CHECK_CUDA(cudaGetLastError());
    note_launch();
  }
  return 0;
}

extern "C" int lp_lowrank_operand(const float* t, long long ldt, int R, int rank, int act_tanh, void* out, long long ldo, int split,
                                  void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(t != nullptr && out != nullptr && R >= 0 && rank > 0 && ldo >= (split ? 2 : 1) * rank, "lp_lowrank_operand: bad arguments");
  if (R == 0) return 0;
  lowrank_operand_kernel<<<(unsigned)(((long long)R * rank + 255) / 256), 256, 0, stream>>>(
      t, ldt, R, rank, act_tanh, split ? nullptr : reinterpret_cast<float*>(out), split ? reinterpret_cast<bf16*>(out) : nullptr, ldo);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}
