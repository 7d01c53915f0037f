// leopard_b200 — glue kernels of models whose residual stream is kept in 32-bit floats.
//
//   lp_embed_rows_f32   x[r, :] = table[ids[r], :] * scale  (bf16 table -> fp32 rows)
//   lp_rmsnorm_f32      y = x / sqrt(mean(x^2) + eps) * g over fp32 rows, eps inside the root; g is one number (gain_scalar), a vector
//                       (gain_vec) or both.  The result is written as fp32 or bf16 (the operand of the next matrix product), or — with
//                       `accum` — added to another fp32 matrix: the sandwich-norm residual update x <- x + norm(sublayer(x)) in one pass.
//   lp_glu_f32          elementwise epilogues for matrix products that ran elsewhere: xIELU, squared relu, silu(gate) * up, gelu(gate) * up.
//   lp_axpy_f32         y <- y + alpha x, the residual update after such a product.
//   lp_add_positions_f32  x[r, 2i] += sin(p f_i), x[r, 2i + 1] += cos(p f_i) with p the row's position: absolute sinusoidal positions
//                       added to the stream (fp32 angles with the product's rounding error carried along, accurate sincosf).
//   lp_embed_streams_f32  x[r, s, :] = table[ids[r], :] * scale + pos[p, :]: the embedding with learned positions, written as every copy of a
//                       stream that is kept several times (hyper-connections).
//   lp_hyper_f32        closes one sublayer of a hyper-connected layer, x_t <- sum_s mix[s, t] x_s + out[t] y, and opens the next one, h =
//                       norm(sum_s in[s] x_s), in one pass over the copies; in one-token steps also the token-shifted mixes of h.
//   lp_token_shift_mix_f32  the token shift with several mixing vectors at once: one operand per vector from one read of the rows.
//   lp_add_row_f32      x[r, :] += v for every row (a learned vector that marks a pass of a looped stack).
//   lp_token_shift_f32  y_t = h_t + (h_(t-1) - h_t) * mu per channel, with h the rows as they came in; the row before a request's
//                       first row of this step comes from the request's slot (zeros at position 0), and the slot then takes the
//                       request's last row.
//   lp_causal_conv_f32  out_t = (h_t +) sum_j w_j h_(t - K + 1 + j) per channel: a short causal convolution, added to its input when asked; the K - 1
//                       inputs before a request's first row of this step come from the request's slot (zeros before position 0), and
//                       the slot then takes the request's last K - 1 inputs.
//   lp_post_norm_f32    x <- norm(alpha x + y) * gain, the norm after the residual sum, in place; the same pass writes the next sublayer's
//                       operand: the new x, for one-token steps with the next sublayer's causal convolution applied on the way.
//   lp_dyt_f32          Dynamic Tanh: tanh(alpha x) * gain + shift per element, no statistics; one pass can serve the two sublayers of a
//                       parallel layer (two parameter sets, two outputs).
//   lp_rmsnorm_gated_f32  the RMS norm with a vector gain, multiplied by sigmoid(gate) per element (norm over a mixer's concatenated
//                       heads and its output gate in one pass).
//   lp_gated_axpy_f32   x <- x + mult (y + y_bias) sigmoid(g + g_bias): a residual branch behind a learned gate.
//   lp_depth_average_f32  out = sum_j coef[j] X_j over the results of all layers so far (and a copy of it for the next layer's branches).
//
// One warp per row, statistics and normalisation in fp32; the row is read twice (the second read hits L1 / L2).
#include "lp_host.h"
#include "../../include/leopard_b200.h"

namespace lp {

typedef __nv_bfloat16 bf16;

__global__ void embed_rows_f32_kernel(const int* __restrict__ ids, int R, const bf16* __restrict__ table, long long ldt, int vocab,
                                      float scale, float* __restrict__ out, long long ldo, int D) {
  const int r = blockIdx.x;
  if (r >= R) return;
  int id = ids[r];
  if (id < 0 || id >= vocab) id = 0;   // the host validates ids; this only keeps a bad one inside the table
  const bf16* src = table + (long long)id * ldt;
  float* dst = out + (long long)r * ldo;
  for (int c = threadIdx.x; c < D; c += blockDim.x) dst[c] = __bfloat162float(src[c]) * scale;
}

constexpr int NORM32_WARPS = 8;
__global__ void __launch_bounds__(NORM32_WARPS * 32)
rmsnorm_f32_kernel(const float* __restrict__ x, long long ldx, int M, int D, float gain_scalar, const float* __restrict__ gain_vec,
                   float eps, float* __restrict__ out_f32, bf16* __restrict__ out_bf16, long long ldo, float* __restrict__ accum,
                   long long lda) {
  const int row = blockIdx.x * NORM32_WARPS + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (row >= M) return;
  const float* xr = x + (long long)row * ldx;
  float ss = 0.f;
  for (int c = lane; c < D; c += 32) {
    const float v = xr[c];
    ss = fmaf(v, v, ss);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float r = 1.0f / sqrtf(ss / (float)D + eps);
  for (int c = lane; c < D; c += 32) {
    float v = xr[c] * r * gain_scalar;
    if (gain_vec != nullptr) v *= gain_vec[c];
    if (accum != nullptr) accum[(long long)row * lda + c] += v;
    else if (out_f32 != nullptr) out_f32[(long long)row * ldo + c] = v;
    else out_bf16[(long long)row * ldo + c] = __float2bfloat16(v);
  }
}

template <typename T> __device__ __forceinline__ float ld32(const T* p);
template <> __device__ __forceinline__ float ld32<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ld32<bf16>(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st32(float* p, float v) { *p = v; }
__device__ __forceinline__ void st32(bf16* p, float v) { *p = __float2bfloat16(v); }

// mode LP_EPI_XIELU: out[m, n] = xielu(in[m, n]); LP_EPI_SILU_GATE, LP_EPI_GELU_GATE:
// out[m, n] = silu | gelu (in[m, n]) * in[m, n + N]; LP_EPI_CLAMP_GLU: the
// clamped gated unit of lp_linear on (in[m, n], in[m, n + N]) with limit a and slope b.  row_scale multiplies what is read.
template <typename IT, typename OT>
__global__ void glu_kernel(const IT* __restrict__ in, long long ldi, OT* __restrict__ out, long long ldo, int M, int N, int mode, float a,
                           float b, const float* __restrict__ row_scale) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)M * N) return;
  const int m = (int)(i / N), n = (int)(i % N);
  const float rs = row_scale != nullptr ? row_scale[m] : 1.0f;
  const float z = ld32<IT>(in + (long long)m * ldi + n) * rs;
  float v;
  if (mode == LP_EPI_SILU_GATE) v = z / (1.0f + expf(-z)) * (ld32<IT>(in + (long long)m * ldi + n + N) * rs);
  else if (mode == LP_EPI_GELU_GATE) {      // tanh form: 1/2 (1 + tanh t) = sigmoid(2 t) with t = sqrt(2 / pi) (z + 0.044715 z^3)
    const float t = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
    v = z / (1.0f + expf(-2.0f * t)) * (ld32<IT>(in + (long long)m * ldi + n + N) * rs);
  }
  else if (mode == LP_EPI_CLAMP_GLU) {
    const float g = fminf(z, a), u = fminf(fmaxf(ld32<IT>(in + (long long)m * ldi + n + N) * rs, -a), a);
    v = g / (1.0f + expf(-b * g)) * (u + 1.0f);
  }
  else if (mode == LP_EPI_RELU2) v = fmaxf(z, 0.f) * fmaxf(z, 0.f);
  else v = z > 0.f ? a * z * z + 0.5f * z : b * (expm1f(z) - z) + 0.5f * z;
  st32(out + (long long)m * ldo + n, v);
}

// The three elementwise kernels below work on groups of V consecutive columns per thread: V = 4 (16-byte fp32 accesses, 8-byte bf16
// stores) when the width and every row stride and base allow it, else V = 1.
template <int V> struct f32vec;
template <> struct f32vec<1> { float v[1]; };
template <> struct alignas(16) f32vec<4> { float v[4]; };
template <int V> __device__ __forceinline__ f32vec<V> ldv(const float* p) { return *reinterpret_cast<const f32vec<V>*>(p); }
template <int V> __device__ __forceinline__ void stv(float* p, const f32vec<V>& x) { *reinterpret_cast<f32vec<V>*>(p) = x; }
template <int V> __device__ __forceinline__ void stv(bf16* p, const f32vec<V>& x) {
  if constexpr (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(x.v[0], x.v[1]), hi = __floats2bfloat162_rn(x.v[2], x.v[3]);
    uint2 u;
    u.x = *reinterpret_cast<const unsigned*>(&lo);
    u.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
  } else {
    *p = __float2bfloat16(x.v[0]);
  }
}

// a warp per row; the lanes take groups of V consecutive columns (V = 4: 16-byte reads of the row and of its gate)
template <typename OT, int V>
__global__ void __launch_bounds__(NORM32_WARPS * 32)
rmsnorm_gated_f32_kernel(const float* __restrict__ x, long long ldx, int M, int D, const float* __restrict__ gain, float eps,
                         const float* __restrict__ gate, long long ldg, OT* __restrict__ out, long long ldo) {
  const int row = blockIdx.x * NORM32_WARPS + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (row >= M) return;
  const float* xr = x + (long long)row * ldx;
  float ss = 0.f;
  for (int c = lane * V; c < D; c += 32 * V) {
    const f32vec<V> v = ldv<V>(xr + c);
#pragma unroll
    for (int k = 0; k < V; ++k) ss = fmaf(v.v[k], v.v[k], ss);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float r = 1.0f / sqrtf(ss / (float)D + eps);
  for (int c = lane * V; c < D; c += 32 * V) {
    f32vec<V> v = ldv<V>(xr + c);
    const f32vec<V> g = ldv<V>(gate + (long long)row * ldg + c);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      v.v[k] *= r;
      if (gain != nullptr) v.v[k] *= gain[c + k];
      v.v[k] /= 1.0f + expf(-g.v[k]);
    }
    stv<V>(out + (long long)row * ldo + c, v);
  }
}

// tanh for an output that is rounded to bf16 (8 bits of mantissa): 1 - 2 / (e^(2|x|) + 1) on the fast exponential and division
// (absolute error of a few 1e-7, far below the rounding that follows); the fp32 output keeps the accurate tanhf
template <typename OT> __device__ __forceinline__ float dyt_tanh(float x);
template <> __device__ __forceinline__ float dyt_tanh<float>(float x) { return tanhf(x); }
template <> __device__ __forceinline__ float dyt_tanh<bf16>(float x) {
  const float a = fminf(fabsf(x), 15.f);      // tanh(15) rounds to 1 in fp32; the bound keeps the exponential finite
  const float t = 1.0f - __fdividef(2.0f, __expf(2.0f * a) + 1.0f);
  return copysignf(t, x);
}

template <typename OT, int V>
__global__ void dyt_f32_kernel(const float* __restrict__ x, long long ldx, int M, int D, float alpha, const float* __restrict__ gain,
                               const float* __restrict__ shift, OT* __restrict__ out, long long ldo, float alpha2,
                               const float* __restrict__ gain2, const float* __restrict__ shift2, OT* __restrict__ out2, long long ldo2) {
  const int DV = D / V;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)M * DV) return;
  const int m = (int)(i / DV), c = (int)(i % DV) * V;
  const f32vec<V> v = ldv<V>(x + (long long)m * ldx + c);
  f32vec<V> y;
  {
    const f32vec<V> g = ldv<V>(gain + c);
#pragma unroll
    for (int k = 0; k < V; ++k) y.v[k] = fmaf(dyt_tanh<OT>(alpha * v.v[k]), g.v[k], shift != nullptr ? shift[c + k] : 0.f);
    stv<V>(out + (long long)m * ldo + c, y);
  }
  if (out2 != nullptr) {
    const f32vec<V> g = ldv<V>(gain2 + c);
#pragma unroll
    for (int k = 0; k < V; ++k) y.v[k] = fmaf(dyt_tanh<OT>(alpha2 * v.v[k]), g.v[k], shift2 != nullptr ? shift2[c + k] : 0.f);
    stv<V>(out2 + (long long)m * ldo2 + c, y);
  }
}

template <int V>
__global__ void gated_axpy_f32_kernel(float* __restrict__ x, long long ldx, const float* __restrict__ y, long long ldy,
                                      const float* __restrict__ y_bias, const float* __restrict__ g, long long ldg,
                                      const float* __restrict__ g_bias, float mult, int M, int N) {
  const int NV = N / V;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)M * NV) return;
  const int m = (int)(i / NV), n = (int)(i % NV) * V;
  f32vec<V> acc = ldv<V>(x + (long long)m * ldx + n);
  const f32vec<V> yv = ldv<V>(y + (long long)m * ldy + n);
  f32vec<V> gv;
  if (g != nullptr) gv = ldv<V>(g + (long long)m * ldg + n);
#pragma unroll
  for (int k = 0; k < V; ++k) {
    float v = yv.v[k] + (y_bias != nullptr ? y_bias[n + k] : 0.f);
    if (g != nullptr) v /= 1.0f + expf(-(gv.v[k] + (g_bias != nullptr ? g_bias[n + k] : 0.f)));
    acc.v[k] = fmaf(mult, v, acc.v[k]);
  }
  stv<V>(x + (long long)m * ldx + n, acc);
}

template <int V>
__global__ void depth_average_f32_kernel(const float* __restrict__ hist, long long layer_stride, long long ldh,
                                         const float* __restrict__ coef, int n, float* __restrict__ out, long long ldo,
                                         float* __restrict__ copy, long long ldc, int M, int N) {
  const int NV = N / V;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)M * NV) return;
  const int m = (int)(i / NV), c = (int)(i % NV) * V;
  const float* src = hist + (long long)m * ldh + c;
  f32vec<V> acc;
#pragma unroll
  for (int k = 0; k < V; ++k) acc.v[k] = 0.f;
  for (int j = 0; j < n; ++j) {
    const f32vec<V> h = ldv<V>(src + (long long)j * layer_stride);
    const float cj = coef[j];
#pragma unroll
    for (int k = 0; k < V; ++k) acc.v[k] = fmaf(cj, h.v[k], acc.v[k]);
  }
  stv<V>(out + (long long)m * ldo + c, acc);
  if (copy != nullptr) stv<V>(copy + (long long)m * ldc + c, acc);
}

// 16-byte accesses need every base on a 16-byte boundary and every row stride a multiple of four floats
static bool vec4_ok(int N, std::initializer_list<const void*> bases, std::initializer_list<long long> strides) {
  if (N % 4) return false;
  for (const void* b : bases)
    if (b != nullptr && (reinterpret_cast<uintptr_t>(b) & 15)) return false;
  for (long long s : strides)
    if (s % 4) return false;
  return true;
}

__global__ void axpy_f32_kernel(float* __restrict__ y, long long ldy, const float* __restrict__ x, long long ldx, float alpha, int M, int N) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)M * N) return;
  const int m = (int)(i / N), n = (int)(i % N);
  y[(long long)m * ldy + n] = fmaf(alpha, x[(long long)m * ldx + n], y[(long long)m * ldy + n]);
}

// pair i of a row: (sin, cos) of position * frequency i; an odd width leaves the last sine without its cosine.  The frequency comes as
// two floats hi + lo (a float64 value split once on the host), and the product's rounding error is recovered with one fma, so the
// angle is a = fl(p hi) plus a small rest e known to about 2^-48 of a: sin(a + e) = sin a + e cos a, cos(a + e) = cos a - e sin a.
__global__ void add_positions_f32_kernel(float* __restrict__ x, long long ldx, int R, int D, const int* __restrict__ row_pos,
                                         const float* __restrict__ freq, int n_freq) {
  const int r = blockIdx.x;
  if (r >= R) return;
  const float p = (float)row_pos[r];
  float* xr = x + (long long)r * ldx;
  for (int i = threadIdx.x; 2 * i < D; i += blockDim.x) {
    const float hi = freq[i], lo = freq[n_freq + i];
    const float a = p * hi;
    const float e = fmaf(p, hi, -a) + p * lo;
    float s, c;
    sincosf(a, &s, &c);
    xr[2 * i] += fmaf(e, c, s);
    if (2 * i + 1 < D) xr[2 * i + 1] += fmaf(-e, s, c);
  }
}

__global__ void add_row_f32_kernel(float* __restrict__ x, long long ldx, const float* __restrict__ v, int M, int N) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)M * N) return;
  const int m = (int)(i / N), n = (int)(i % N);
  x[(long long)m * ldx + n] += v[n];
}

// One thread per (row, channel).  Only the thread of a request's FIRST row touches the request's slot: it reads the carried row
// and then stores the request's last row of this step there, so no other thread of the launch reads what it writes.
template <typename OT>
__global__ void token_shift_kernel(const float* __restrict__ h, long long ldh, const float* __restrict__ mu, int R, int D,
                                   const int* __restrict__ row_seq, const int* __restrict__ row_pos, const int* __restrict__ seq_row0,
                                   const int* __restrict__ seq_slot, float* __restrict__ state, long long slot_stride,
                                   OT* __restrict__ out, long long ldo) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)R * D) return;
  const int r = (int)(i / D), c = (int)(i % D);
  const int s = row_seq[r];
  const float cur = h[(long long)r * ldh + c];
  float prev;
  if (r == seq_row0[s]) {
    float* slot = state + (long long)seq_slot[s] * slot_stride;
    prev = row_pos[r] > 0 ? slot[c] : 0.f;
    slot[c] = h[(long long)(seq_row0[s + 1] - 1) * ldh + c];
  } else {
    prev = h[(long long)(r - 1) * ldh + c];
  }
  st32(out + (long long)r * ldo + c, fmaf(prev - cur, mu[c], cur));
}

// Short causal convolution, added to its input or by itself.  A thread owns V channels of one TILE of consecutive rows of a request and walks the
// rows with the K - 1 inputs before them in registers.  Tiles (and full chunks) are at least K - 1 rows long, so only the thread of a
// request's FIRST tile reaches back past the rows of this step into the request's slot: it reads the carried inputs and then stores
// the request's last K - 1 inputs there, and no other thread of the launch touches them.  The slot holds K - 1 rows of D, oldest
// first, zeros for positions before the request's start.
template <typename OT, int V, int K>
__global__ void causal_conv_kernel(const float* __restrict__ h, long long ldh, const float* __restrict__ w, int D, const int* __restrict__ chunk_seq,
                                   const int* __restrict__ chunk_row0, const int* __restrict__ chunk_len, int subs, int tile,
                                   const int* __restrict__ row_pos, const int* __restrict__ seq_row0, const int* __restrict__ seq_slot,
                                   float* __restrict__ state, long long slot_stride, OT* __restrict__ out, long long ldo, float own) {
  const int ck = blockIdx.x / subs, sub = blockIdx.x % subs;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (sub * tile >= chunk_len[ck] || c >= D) return;
  const int s = chunk_seq[ck], first = seq_row0[s], end = seq_row0[s + 1];
  const int r0 = chunk_row0[ck] + sub * tile, rows = min(tile, chunk_len[ck] - sub * tile);
  const bool started = row_pos[first] > 0;      // earlier steps left inputs in the slot
  float* slot = state + (long long)seq_slot[s] * slot_stride + c;
  f32vec<V> wv[K], win[K];      // win[k]: the input K - 1 - k rows before the current one; win[K - 1] the current one
#pragma unroll
  for (int k = 0; k < K; ++k) {
    wv[k] = ldv<V>(w + (long long)k * D + c);
#pragma unroll
    for (int i = 0; i < V; ++i) win[k].v[i] = 0.f;
  }
#pragma unroll
  for (int k = 0; k < K - 1; ++k) {
    const int r = r0 - (K - 1) + k;
    if (r >= first) win[k] = ldv<V>(h + (long long)r * ldh + c);
    else if (started) win[k] = ldv<V>(slot + (long long)(K - 1 + r - first) * D);
  }
  if (K > 1 && r0 == first) {
    f32vec<V> zero;
#pragma unroll
    for (int i = 0; i < V; ++i) zero.v[i] = 0.f;
    for (int k = 0; k < K - 1; ++k) {      // row end - (K - 1) + k; a carried one moves towards the slot's start, so in place is safe
      const int r = end - (K - 1) + k;
      stv<V>(slot + (long long)k * D, r >= first ? ldv<V>(h + (long long)r * ldh + c) : started ? ldv<V>(slot + (long long)(K - 1 + r - first) * D) : zero);
    }
  }
  for (int t = 0; t < rows; ++t) {
    const long long r = r0 + t;
    win[K - 1] = ldv<V>(h + r * ldh + c);
    f32vec<V> y;
#pragma unroll
    for (int i = 0; i < V; ++i) y.v[i] = own * win[K - 1].v[i];
#pragma unroll
    for (int k = 0; k < K; ++k)
#pragma unroll
      for (int i = 0; i < V; ++i) y.v[i] = fmaf(wv[k].v[i], win[k].v[i], y.v[i]);
    stv<V>(out + r * ldo + c, y);
#pragma unroll
    for (int k = 0; k < K - 1; ++k) win[k] = win[k + 1];
  }
}

// More taps than the register window holds: one channel per thread, every input read again for every tap.  The same ownership of the
// slot, which the thread of a request's first tile rewrites after its last row.
template <typename OT>
__global__ void causal_conv_long_kernel(const float* __restrict__ h, long long ldh, const float* __restrict__ w, int K, int D,
                                        const int* __restrict__ chunk_seq, const int* __restrict__ chunk_row0, const int* __restrict__ chunk_len,
                                        const int* __restrict__ row_pos, const int* __restrict__ seq_row0, const int* __restrict__ seq_slot,
                                        float* state, long long slot_stride, OT* __restrict__ out, long long ldo, float own) {
  const int ck = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= D) return;
  const int s = chunk_seq[ck], first = seq_row0[s], end = seq_row0[s + 1], r0 = chunk_row0[ck];
  const bool started = row_pos[first] > 0;
  float* slot = state + (long long)seq_slot[s] * slot_stride + c;
  auto input = [&](int r) {
    if (r >= first) return h[(long long)r * ldh + c];
    return started ? slot[(long long)(K - 1 + r - first) * D] : 0.f;
  };
  for (int r = r0; r < r0 + chunk_len[ck]; ++r) {
    float y = own * h[(long long)r * ldh + c];
    for (int k = 0; k < K; ++k) y = fmaf(w[(long long)k * D + c], input(r - (K - 1) + k), y);
    st32(out + (long long)r * ldo + c, y);
  }
  if (r0 == first)
    for (int k = 0; k < K - 1; ++k) slot[(long long)k * D] = input(end - (K - 1) + k);      // reads ahead of what it writes
}

// a full chunk is as long as the inputs a row looks back at, so no chunk but a request's first needs the slot
constexpr int CONV_WINDOW_TAPS = 8, CONV_MAX_TAPS = LP_RETENTION_CHUNK + 1, CONV_TILE = 16, CONV_THREADS = 128;

struct ConvLaunch {
  const float* h; long long ldh; const float* w; int D;
  int n_chunks; const int *chunk_seq, *chunk_row0, *chunk_len; int longest;
  const int *row_pos, *seq_row0, *seq_slot;
  float* state; long long slot_stride;
  void* out; long long ldo;
  float own;      // 1: the convolution is added to its input, 0: it stands alone
};

template <typename OT, int V, int K>
static void launch_conv(const ConvLaunch& a, cudaStream_t stream) {
  const int subs = (a.longest + CONV_TILE - 1) / CONV_TILE;
  const int cols = a.D / V, threads = cols >= CONV_THREADS ? CONV_THREADS : (cols + 31) / 32 * 32;
  const dim3 grid(a.n_chunks * subs, (cols + threads - 1) / threads);
  causal_conv_kernel<OT, V, K><<<grid, threads, 0, stream>>>(a.h, a.ldh, a.w, a.D, a.chunk_seq, a.chunk_row0, a.chunk_len, subs, CONV_TILE,
                                                                 a.row_pos, a.seq_row0, a.seq_slot, a.state, a.slot_stride,
                                                                 reinterpret_cast<OT*>(a.out), a.ldo, a.own);
}

template <typename OT, int V>
static void launch_conv_taps(const ConvLaunch& a, int taps, cudaStream_t stream) {
  switch (taps) {
    case 1: launch_conv<OT, V, 1>(a, stream); break;
    case 2: launch_conv<OT, V, 2>(a, stream); break;
    case 3: launch_conv<OT, V, 3>(a, stream); break;
    case 4: launch_conv<OT, V, 4>(a, stream); break;
    case 5: launch_conv<OT, V, 5>(a, stream); break;
    case 6: launch_conv<OT, V, 6>(a, stream); break;
    case 7: launch_conv<OT, V, 7>(a, stream); break;
    case 8: launch_conv<OT, V, 8>(a, stream); break;
    default:
      causal_conv_long_kernel<OT><<<dim3(a.n_chunks, (a.D + CONV_THREADS - 1) / CONV_THREADS), CONV_THREADS, 0, stream>>>(
          a.h, a.ldh, a.w, taps, a.D, a.chunk_seq, a.chunk_row0, a.chunk_len, a.row_pos, a.seq_row0, a.seq_slot, a.state, a.slot_stride,
          reinterpret_cast<OT*>(a.out), a.ldo, a.own);
      break;
  }
}

// One CTA per row: x <- norm(alpha x + y) * gain, and the next sublayer's operand.  The sums alpha x + y of the first POST_KEEP column groups
// of a thread stay in registers between the two passes; wider rows park theirs in x.  With conv_w (one-token steps: row m is the only
// row of request m) the operand is the new x plus the causal convolution over the slot's carried inputs and the new x, and the slot
// moves on by one row; a thread reads and writes its own columns of the slot only.
constexpr int POST_THREADS = 256, POST_KEEP = 4;
template <typename OT, int V>
__global__ void __launch_bounds__(POST_THREADS)
post_norm_kernel(float* __restrict__ x, long long ldx, const float* __restrict__ y, long long ldy, float alpha, int D,
                 const float* __restrict__ gain, float eps, OT* __restrict__ out, long long ldo, const float* __restrict__ conv_w, int taps,
                 const int* __restrict__ row_pos, const int* __restrict__ row_slot, float* __restrict__ state, long long slot_stride) {
  __shared__ float red[POST_THREADS / 32];
  const long long m = blockIdx.x;
  const int tid = threadIdx.x, step = blockDim.x * V;
  float* xr = x + m * ldx;
  const float* yr = y + m * ldy;
  f32vec<V> keep[POST_KEEP];
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < POST_KEEP; ++it) {
    const int c = tid * V + it * step;
    if (c < D) {
      const f32vec<V> a = ldv<V>(xr + c), b = ldv<V>(yr + c);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        keep[it].v[i] = fmaf(alpha, a.v[i], b.v[i]);
        ss = fmaf(keep[it].v[i], keep[it].v[i], ss);
      }
    }
  }
  for (int c = tid * V + POST_KEEP * step; c < D; c += step) {
    f32vec<V> a = ldv<V>(xr + c);
    const f32vec<V> b = ldv<V>(yr + c);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      a.v[i] = fmaf(alpha, a.v[i], b.v[i]);
      ss = fmaf(a.v[i], a.v[i], ss);
    }
    stv<V>(xr + c, a);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float total = 0.f;
  for (int k = 0; k < (int)(blockDim.x >> 5); ++k) total += red[k];
  const float r = 1.0f / sqrtf(total / (float)D + eps);
  float* slot = nullptr;
  bool started = false;
  if (conv_w != nullptr && taps > 1) {
    slot = state + (long long)row_slot[m] * slot_stride;
    started = row_pos[m] > 0;
  }
  auto finish = [&](int c, f32vec<V> z) {
    const f32vec<V> g = ldv<V>(gain + c);
#pragma unroll
    for (int i = 0; i < V; ++i) z.v[i] = z.v[i] * r * g.v[i];
    stv<V>(xr + c, z);
    if (out == nullptr) return;
    f32vec<V> o = z;
    if (conv_w != nullptr) {
      for (int k = 0; k < taps - 1; ++k) {
        f32vec<V> old;
#pragma unroll
        for (int i = 0; i < V; ++i) old.v[i] = 0.f;
        if (started) old = ldv<V>(slot + (long long)k * D + c);
        const f32vec<V> wk = ldv<V>(conv_w + (long long)k * D + c);
#pragma unroll
        for (int i = 0; i < V; ++i) o.v[i] = fmaf(wk.v[i], old.v[i], o.v[i]);
        if (k > 0) stv<V>(slot + (long long)(k - 1) * D + c, old);
      }
      const f32vec<V> wk = ldv<V>(conv_w + (long long)(taps - 1) * D + c);
#pragma unroll
      for (int i = 0; i < V; ++i) o.v[i] = fmaf(wk.v[i], z.v[i], o.v[i]);
      if (taps > 1) stv<V>(slot + (long long)(taps - 2) * D + c, z);
    }
    stv<V>(out + m * ldo + c, o);
  };
#pragma unroll
  for (int it = 0; it < POST_KEEP; ++it) {
    const int c = tid * V + it * step;
    if (c < D) finish(c, keep[it]);
  }
  for (int c = tid * V + POST_KEEP * step; c < D; c += step) finish(c, ldv<V>(xr + c));
}

// The embedding with learned positions, written `copies` times side by side (row stride ldo >= copies * D)
__global__ void embed_streams_kernel(const int* __restrict__ ids, int R, const bf16* __restrict__ table, long long ldt, int vocab, float scale,
                                     const bf16* __restrict__ pos_table, long long ldp, int n_pos, const int* __restrict__ row_pos,
                                     float* __restrict__ out, long long ldo, int D, int copies) {
  const int r = blockIdx.x;
  if (r >= R) return;
  int id = ids[r];
  if (id < 0 || id >= vocab) id = 0;   // the host validates ids and positions; this only keeps a bad one inside the tables
  const bf16* src = table + (long long)id * ldt;
  const bf16* pv = nullptr;
  if (pos_table != nullptr) {
    const int p = row_pos[r];
    pv = pos_table + (long long)(p < n_pos ? p : n_pos - 1) * ldp;
  }
  float* dst = out + (long long)r * ldo;
  for (int c = threadIdx.x; c < D; c += blockDim.x) {
    const float v = fmaf(__bfloat162float(src[c]), scale, pv != nullptr ? __bfloat162float(pv[c]) : 0.f);
    for (int s = 0; s < copies; ++s) dst[(long long)s * D + c] = v;
  }
}

// Token shift with n mixing vectors.  One thread per (row, V channels); the slot is touched by the thread of a request's first row only,
// as in token_shift_kernel.
template <typename OT, int V>
__global__ void token_shift_mix_kernel(const float* __restrict__ h, long long ldh, const float* __restrict__ mu, int n, int R, int D,
                                       const int* __restrict__ row_seq, const int* __restrict__ row_pos, const int* __restrict__ seq_row0,
                                       const int* __restrict__ seq_slot, float* __restrict__ state, long long slot_stride,
                                       OT* __restrict__ out, long long ldo, long long mix_stride) {
  const int DV = D / V;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)R * DV) return;
  const int r = (int)(i / DV), c = (int)(i % DV) * V;
  const int s = row_seq[r];
  const f32vec<V> cur = ldv<V>(h + (long long)r * ldh + c);
  f32vec<V> step;
#pragma unroll
  for (int k = 0; k < V; ++k) step.v[k] = 0.f;
  if (r == seq_row0[s]) {
    float* slot = state + (long long)seq_slot[s] * slot_stride + c;
    if (row_pos[r] > 0) step = ldv<V>(slot);
    stv<V>(slot, ldv<V>(h + (long long)(seq_row0[s + 1] - 1) * ldh + c));
  } else {
    step = ldv<V>(h + (long long)(r - 1) * ldh + c);
  }
#pragma unroll
  for (int k = 0; k < V; ++k) step.v[k] -= cur.v[k];
  for (int m = 0; m < n; ++m) {
    const f32vec<V> w = ldv<V>(mu + (long long)m * D + c);
    f32vec<V> y;
#pragma unroll
    for (int k = 0; k < V; ++k) y.v[k] = fmaf(step.v[k], w.v[k], cur.v[k]);
    stv<V>(out + m * mix_stride + (long long)r * ldo + c, y);
  }
}

// Hyper-connections: one CTA per row.  The row's copies x_0 .. x_(n-1) lie side by side.  With y the sublayer before is closed (every copy
// from the old ones), with gain the next one is opened: u = sum_s in[s] x_s is kept in registers for the first HYPER_KEEP column groups of
// a thread (and made again from the copies beyond them) while the row's mean square is summed.  S: the number of copies, 0: any number
// up to HYPER_MAX.  With mu (one-token steps: row m is the only row of request m) the operands are h + (h' - h) * mu_i, h' the row
// carried in the request's slot (zeros at position 0), and the slot then takes h; a thread reads and writes its own columns only.
constexpr int HYPER_THREADS = 256, HYPER_KEEP = 4, HYPER_MAX = 32;
struct HyperArgs {
  float* x; long long ldx; int n, D;
  const float* y; long long ldy; const float* mix; const float* out_w;
  const float* in_w; const float* gain; float eps;
  void* h; long long ldh;
  const float* mu; int n_mix; long long mix_stride;
  const int* row_pos; const int* row_slot; float* state; long long slot_stride;
};
template <typename OT, int V, int S>
__global__ void __launch_bounds__(HYPER_THREADS)
hyper_kernel(HyperArgs a) {
  constexpr int CAP = S > 0 ? S : HYPER_MAX;
  __shared__ float mix_s[CAP * CAP], out_s[CAP], in_s[CAP], red[HYPER_THREADS / 32];
  const int n = S > 0 ? S : a.n;
  const long long m = blockIdx.x;
  const int tid = threadIdx.x, step = blockDim.x * V, D = a.D;
  for (int i = tid; i < n * n; i += blockDim.x) mix_s[i] = a.y != nullptr ? a.mix[i] : 0.f;
  for (int i = tid; i < n; i += blockDim.x) {
    out_s[i] = a.y != nullptr ? a.out_w[i] : 0.f;
    in_s[i] = a.gain != nullptr ? (a.in_w != nullptr ? a.in_w[i] : 1.f) : 0.f;
  }
  __syncthreads();
  float* xr = a.x + m * a.ldx;
  const float* yr = a.y != nullptr ? a.y + m * a.ldy : nullptr;
  f32vec<V> keep[HYPER_KEEP];
  float ss = 0.f;
  auto advance = [&](int c) {      // columns c .. c + V - 1: close, and the sum the next sublayer reads
    f32vec<V> x[CAP], u;
#pragma unroll
    for (int s = 0; s < n; ++s) x[s] = ldv<V>(xr + (long long)s * D + c);
#pragma unroll
    for (int i = 0; i < V; ++i) u.v[i] = 0.f;
    if (yr != nullptr) {
      const f32vec<V> yv = ldv<V>(yr + c);
#pragma unroll
      for (int t = 0; t < n; ++t) {
        f32vec<V> z;
#pragma unroll
        for (int i = 0; i < V; ++i) z.v[i] = out_s[t] * yv.v[i];
#pragma unroll
        for (int s = 0; s < n; ++s)
#pragma unroll
          for (int i = 0; i < V; ++i) z.v[i] = fmaf(mix_s[s * n + t], x[s].v[i], z.v[i]);
        stv<V>(xr + (long long)t * D + c, z);
#pragma unroll
        for (int i = 0; i < V; ++i) u.v[i] = fmaf(in_s[t], z.v[i], u.v[i]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < n; ++s)
#pragma unroll
        for (int i = 0; i < V; ++i) u.v[i] = fmaf(in_s[s], x[s].v[i], u.v[i]);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) ss = fmaf(u.v[i], u.v[i], ss);
    return u;
  };
#pragma unroll
  for (int it = 0; it < HYPER_KEEP; ++it) {
    const int c = tid * V + it * step;
    if (c < D) keep[it] = advance(c);
  }
  for (int c = tid * V + HYPER_KEEP * step; c < D; c += step) advance(c);
  if (a.gain == nullptr) return;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float total = 0.f;
  for (int k = 0; k < (int)(blockDim.x >> 5); ++k) total += red[k];
  const float r = 1.0f / sqrtf(total / (float)D + a.eps);
  float* slot = a.mu != nullptr ? a.state + (long long)a.row_slot[m] * a.slot_stride : nullptr;
  const bool started = a.mu != nullptr && a.row_pos[m] > 0;
  OT* hr = reinterpret_cast<OT*>(a.h) + m * a.ldh;
  auto finish = [&](int c, f32vec<V> u) {
    const f32vec<V> g = ldv<V>(a.gain + c);
#pragma unroll
    for (int i = 0; i < V; ++i) u.v[i] = u.v[i] * r * g.v[i];
    if (a.mu == nullptr) {
      stv<V>(hr + c, u);
      return;
    }
    f32vec<V> prev;
#pragma unroll
    for (int i = 0; i < V; ++i) prev.v[i] = 0.f;
    if (started) prev = ldv<V>(slot + c);
    stv<V>(slot + c, u);
    for (int k = 0; k < a.n_mix; ++k) {
      const f32vec<V> w = ldv<V>(a.mu + (long long)k * D + c);
      f32vec<V> o;
#pragma unroll
      for (int i = 0; i < V; ++i) o.v[i] = fmaf(prev.v[i] - u.v[i], w.v[i], u.v[i]);
      stv<V>(hr + k * a.mix_stride + c, o);
    }
  };
#pragma unroll
  for (int it = 0; it < HYPER_KEEP; ++it) {
    const int c = tid * V + it * step;
    if (c < D) finish(c, keep[it]);
  }
  for (int c = tid * V + HYPER_KEEP * step; c < D; c += step) {
    f32vec<V> u;
#pragma unroll
    for (int i = 0; i < V; ++i) u.v[i] = 0.f;
    for (int s = 0; s < n; ++s) {
      const f32vec<V> x = ldv<V>(xr + (long long)s * D + c);
#pragma unroll
      for (int i = 0; i < V; ++i) u.v[i] = fmaf(in_s[s], x.v[i], u.v[i]);
    }
    finish(c, u);
  }
}

template <typename OT, int V>
static void launch_hyper(const HyperArgs& a, int M, int threads, cudaStream_t stream) {
  switch (a.n) {
    case 1: hyper_kernel<OT, V, 1><<<M, threads, 0, stream>>>(a); break;
    case 2: hyper_kernel<OT, V, 2><<<M, threads, 0, stream>>>(a); break;
    case 3: hyper_kernel<OT, V, 3><<<M, threads, 0, stream>>>(a); break;
    case 4: hyper_kernel<OT, V, 4><<<M, threads, 0, stream>>>(a); break;
    default: hyper_kernel<OT, V, 0><<<M, threads, 0, stream>>>(a); break;
  }
}

}  // namespace lp

using namespace lp;

extern "C" int lp_embed_streams_f32(const int* ids, int R, const void* table, long long ldt, int vocab, float scale, const void* pos_table,
                                    long long ldp, int n_pos, const int* row_pos, float* out, long long ldo, int D, int copies, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(ids != nullptr && table != nullptr && out != nullptr && R >= 0 && D > 0 && vocab > 0 && copies > 0 && ldo >= (long long)copies * D,
             "lp_embed_streams_f32: bad arguments");
  LP_REQUIRE(pos_table == nullptr || (n_pos > 0 && row_pos != nullptr), "lp_embed_streams_f32: a position table without positions");
  if (R == 0) return 0;
  embed_streams_kernel<<<R, 128, 0, stream>>>(ids, R, reinterpret_cast<const bf16*>(table), ldt, vocab, scale,
                                              reinterpret_cast<const bf16*>(pos_table), ldp, n_pos, row_pos, out, ldo, D, copies);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_token_shift_mix_f32(const float* h, long long ldh, const float* mu, int n, int R, int D, const int* row_seq,
                                      const int* row_pos, const int* seq_row0, const int* seq_slot, float* state, long long slot_stride,
                                      void* out, long long ldo, long long mix_stride, int out_fp32, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(h != nullptr && mu != nullptr && out != nullptr && state != nullptr && row_seq != nullptr && row_pos != nullptr &&
                 seq_row0 != nullptr && seq_slot != nullptr && n > 0 && R >= 0 && D > 0 && slot_stride >= D,
             "lp_token_shift_mix_f32: bad arguments");
  LP_REQUIRE(h != out, "lp_token_shift_mix_f32: a row reads its neighbour as it came in, so it cannot run in place");
  if (R == 0) return 0;
  const bool v4 = vec4_ok(D, {h, mu, state, out}, {ldh, slot_stride, ldo, mix_stride});
  const unsigned grid = (unsigned)(((long long)R * (v4 ? D / 4 : D) + 255) / 256);
  if (out_fp32 && v4)
    token_shift_mix_kernel<float, 4><<<grid, 256, 0, stream>>>(h, ldh, mu, n, R, D, row_seq, row_pos, seq_row0, seq_slot, state, slot_stride,
                                                               reinterpret_cast<float*>(out), ldo, mix_stride);
  else if (out_fp32)
    token_shift_mix_kernel<float, 1><<<grid, 256, 0, stream>>>(h, ldh, mu, n, R, D, row_seq, row_pos, seq_row0, seq_slot, state, slot_stride,
                                                               reinterpret_cast<float*>(out), ldo, mix_stride);
  else if (v4)
    token_shift_mix_kernel<bf16, 4><<<grid, 256, 0, stream>>>(h, ldh, mu, n, R, D, row_seq, row_pos, seq_row0, seq_slot, state, slot_stride,
                                                              reinterpret_cast<bf16*>(out), ldo, mix_stride);
  else
    token_shift_mix_kernel<bf16, 1><<<grid, 256, 0, stream>>>(h, ldh, mu, n, R, D, row_seq, row_pos, seq_row0, seq_slot, state, slot_stride,
                                                              reinterpret_cast<bf16*>(out), ldo, mix_stride);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_hyper_max_streams(void) { return HYPER_MAX; }

extern "C" int lp_hyper_f32(const lp_hyper_desc* d, int M, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(d != nullptr && d->x != nullptr && d->n >= 1 && d->n <= HYPER_MAX && d->D > 0 && M >= 0 && d->ldx >= (long long)d->n * d->D,
             "lp_hyper_f32: bad arguments (1 .. %d streams)", HYPER_MAX);
  LP_REQUIRE(d->y == nullptr || (d->mix != nullptr && d->out_w != nullptr), "lp_hyper_f32: a result without its connection weights");
  LP_REQUIRE((d->gain != nullptr) == (d->h != nullptr) && (d->y != nullptr || d->gain != nullptr), "lp_hyper_f32: nothing to do");
  LP_REQUIRE(d->mu == nullptr || (d->gain != nullptr && d->n_mix > 0 && d->row_pos != nullptr && d->row_slot != nullptr && d->state != nullptr &&
                                  d->slot_stride >= d->D),
             "lp_hyper_f32: a token shift without its slot");
  if (M == 0) return 0;
  HyperArgs a{d->x, d->ldx, d->n, d->D, d->y, d->ldy, d->mix, d->out_w, d->in_w, d->gain, d->eps, d->h, d->ldh, d->mu, d->n_mix,
              d->mix_stride, d->row_pos, d->row_slot, d->state, d->slot_stride};
  const bool v4 = vec4_ok(d->D, {d->x, d->y, d->gain, d->h, d->mu, d->state},
                          {d->ldx, d->y != nullptr ? d->ldy : 0, d->h != nullptr ? d->ldh : 0, d->mu != nullptr ? d->mix_stride : 0,
                           d->state != nullptr ? d->slot_stride : 0});
  int threads = v4 ? d->D / 4 : d->D;
  threads = threads >= HYPER_THREADS ? HYPER_THREADS : (threads + 31) / 32 * 32;
  if (d->h_fp32 && v4) launch_hyper<float, 4>(a, M, threads, stream);
  else if (d->h_fp32) launch_hyper<float, 1>(a, M, threads, stream);
  else if (v4) launch_hyper<bf16, 4>(a, M, threads, stream);
  else launch_hyper<bf16, 1>(a, M, threads, stream);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_causal_conv_max_taps(void) { return CONV_MAX_TAPS; }

extern "C" int lp_causal_conv_f32(const float* h, long long ldh, const float* w, int taps, int add_input, int D, int n_chunks, const int* chunk_seq,
                                  const int* chunk_row0, const int* chunk_len, int longest_chunk, const int* row_pos, const int* seq_row0,
                                  const int* seq_slot, float* state, long long slot_stride, void* out, long long ldo, int out_fp32,
                                  void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(h != nullptr && w != nullptr && out != nullptr && chunk_seq != nullptr && chunk_row0 != nullptr && chunk_len != nullptr &&
                 row_pos != nullptr && seq_row0 != nullptr && seq_slot != nullptr && D > 0 && n_chunks >= 0,
             "lp_causal_conv_f32: bad arguments");
  LP_REQUIRE(taps >= 1 && taps <= CONV_MAX_TAPS, "lp_causal_conv_f32: %d taps (1 .. %d are built)", taps, CONV_MAX_TAPS);
  LP_REQUIRE(taps == 1 || (state != nullptr && slot_stride >= (long long)(taps - 1) * D), "lp_causal_conv_f32: no room for the carried inputs");
  LP_REQUIRE(longest_chunk >= 1 && longest_chunk <= LP_RETENTION_CHUNK, "lp_causal_conv_f32: longest_chunk=%d", longest_chunk);
  LP_REQUIRE(h != out, "lp_causal_conv_f32: a row reads its neighbours as they came in, so it cannot run in place");
  if (n_chunks == 0) return 0;
  const ConvLaunch a{h, ldh, w, D, n_chunks, chunk_seq, chunk_row0, chunk_len, longest_chunk, row_pos, seq_row0, seq_slot, state, slot_stride, out, ldo,
                     add_input ? 1.f : 0.f};
  const bool v4 = taps <= CONV_WINDOW_TAPS && vec4_ok(D, {h, w, state, out}, {ldh, ldo, taps > 1 ? slot_stride : 0});
  if (out_fp32 && v4) launch_conv_taps<float, 4>(a, taps, stream);
  else if (out_fp32) launch_conv_taps<float, 1>(a, taps, stream);
  else if (v4) launch_conv_taps<bf16, 4>(a, taps, stream);
  else launch_conv_taps<bf16, 1>(a, taps, stream);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_post_norm_f32(float* x, long long ldx, const float* y, long long ldy, float alpha, int M, int D, const float* gain, float eps,
                                void* out, long long ldo, int out_fp32, const float* conv_w, int taps, const int* row_pos,
                                const int* row_slot, float* state, long long slot_stride, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(x != nullptr && y != nullptr && gain != nullptr && M >= 0 && D > 0, "lp_post_norm_f32: bad arguments");
  LP_REQUIRE(conv_w == nullptr || (out != nullptr && taps >= 1), "lp_post_norm_f32: a convolution without its operand");
  LP_REQUIRE(conv_w == nullptr || taps == 1 ||
                 (row_pos != nullptr && row_slot != nullptr && state != nullptr && slot_stride >= (long long)(taps - 1) * D),
             "lp_post_norm_f32: no room for the carried inputs");
  LP_REQUIRE(out != x, "lp_post_norm_f32: the operand needs memory of its own");
  if (M == 0) return 0;
  const bool v4 = vec4_ok(D, {x, y, gain, out, conv_w, state}, {ldx, ldy, out != nullptr ? ldo : 0, state != nullptr ? slot_stride : 0});
  int threads = (v4 ? D / 4 : D);
  threads = threads >= POST_THREADS ? POST_THREADS : (threads + 31) / 32 * 32;
  if (out_fp32 && v4)
    post_norm_kernel<float, 4><<<M, threads, 0, stream>>>(x, ldx, y, ldy, alpha, D, gain, eps, reinterpret_cast<float*>(out), ldo, conv_w, taps,
                                                          row_pos, row_slot, state, slot_stride);
  else if (out_fp32)
    post_norm_kernel<float, 1><<<M, threads, 0, stream>>>(x, ldx, y, ldy, alpha, D, gain, eps, reinterpret_cast<float*>(out), ldo, conv_w, taps,
                                                          row_pos, row_slot, state, slot_stride);
  else if (v4)
    post_norm_kernel<bf16, 4><<<M, threads, 0, stream>>>(x, ldx, y, ldy, alpha, D, gain, eps, reinterpret_cast<bf16*>(out), ldo, conv_w, taps,
                                                         row_pos, row_slot, state, slot_stride);
  else
    post_norm_kernel<bf16, 1><<<M, threads, 0, stream>>>(x, ldx, y, ldy, alpha, D, gain, eps, reinterpret_cast<bf16*>(out), ldo, conv_w, taps,
                                                         row_pos, row_slot, state, slot_stride);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_add_positions_f32(float* x, long long ldx, int R, int D, const int* row_pos, const float* freq, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(x != nullptr && row_pos != nullptr && freq != nullptr && R >= 0 && D > 0, "lp_add_positions_f32: bad arguments");
  if (R == 0) return 0;
  add_positions_f32_kernel<<<R, 128, 0, stream>>>(x, ldx, R, D, row_pos, freq, (D + 1) / 2);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_add_row_f32(float* x, long long ldx, const float* v, int M, int N, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(x != nullptr && v != nullptr && M >= 0 && N > 0, "lp_add_row_f32: bad arguments");
  if (M == 0) return 0;
  add_row_f32_kernel<<<(unsigned)(((long long)M * N + 255) / 256), 256, 0, stream>>>(x, ldx, v, M, N);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_token_shift_f32(const float* h, long long ldh, const float* mu, int R, int D, const int* row_seq, const int* row_pos,
                                  const int* seq_row0, const int* seq_slot, float* state, long long slot_stride, void* out,
                                  long long ldo, int out_fp32, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(h != nullptr && mu != nullptr && out != nullptr && state != nullptr && row_seq != nullptr && row_pos != nullptr &&
                 seq_row0 != nullptr && seq_slot != nullptr && R >= 0 && D > 0 && slot_stride >= D,
             "lp_token_shift_f32: bad arguments");
  LP_REQUIRE(h != out, "lp_token_shift_f32: a row reads its neighbour as it came in, so it cannot run in place");
  if (R == 0) return 0;
  const unsigned grid = (unsigned)(((long long)R * D + 255) / 256);
  if (out_fp32)
    token_shift_kernel<float><<<grid, 256, 0, stream>>>(h, ldh, mu, R, D, row_seq, row_pos, seq_row0, seq_slot, state, slot_stride,
                                                        reinterpret_cast<float*>(out), ldo);
  else
    token_shift_kernel<bf16><<<grid, 256, 0, stream>>>(h, ldh, mu, R, D, row_seq, row_pos, seq_row0, seq_slot, state, slot_stride,
                                                       reinterpret_cast<bf16*>(out), ldo);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_embed_rows_f32(const int* ids, int R, const void* table, long long ldt, int vocab, float scale, float* out, long long ldo,
                                 int D, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(ids != nullptr && table != nullptr && out != nullptr && R >= 0 && D > 0 && vocab > 0, "lp_embed_rows_f32: bad arguments");
  if (R == 0) return 0;
  embed_rows_f32_kernel<<<R, 128, 0, stream>>>(ids, R, reinterpret_cast<const bf16*>(table), ldt, vocab, scale, out, ldo, D);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_rmsnorm_f32(const float* x, long long ldx, int M, int D, float gain_scalar, const float* gain_vec, float eps, void* out,
                              long long ldo, int out_fp32, float* accum, long long ld_accum, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(x != nullptr && M >= 0 && D > 0, "lp_rmsnorm_f32: bad arguments");
  LP_REQUIRE((out != nullptr) != (accum != nullptr), "lp_rmsnorm_f32: give either `out` or `accum`");
  if (M == 0) return 0;
  rmsnorm_f32_kernel<<<(M + NORM32_WARPS - 1) / NORM32_WARPS, NORM32_WARPS * 32, 0, stream>>>(
      x, ldx, M, D, gain_scalar, gain_vec, eps, (out != nullptr && out_fp32) ? reinterpret_cast<float*>(out) : nullptr,
      (out != nullptr && !out_fp32) ? reinterpret_cast<bf16*>(out) : nullptr, ldo, accum, ld_accum);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_glu_f32(const void* in, long long ldi, int in_fp32, void* out, long long ldo, int out_fp32, int M, int N, int mode,
                          float a, float b, void* stream_) {
  return lp_glu_scaled_f32(in, ldi, in_fp32, out, ldo, out_fp32, M, N, mode, a, b, nullptr, stream_);
}

extern "C" int lp_glu_scaled_f32(const void* in, long long ldi, int in_fp32, void* out, long long ldo, int out_fp32, int M, int N, int mode,
                                 float a, float b, const float* row_scale, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(in != nullptr && out != nullptr && M >= 0 && N > 0, "lp_glu_f32: bad arguments");
  LP_REQUIRE(mode == LP_EPI_XIELU || mode == LP_EPI_SILU_GATE || mode == LP_EPI_RELU2 || mode == LP_EPI_CLAMP_GLU ||
                 mode == LP_EPI_GELU_GATE,
             "lp_glu_f32: mode %d is not an activation", mode);
  if (M == 0) return 0;
  const unsigned grid = (unsigned)(((long long)M * N + 255) / 256);
  if (in_fp32 && out_fp32)
    glu_kernel<float, float><<<grid, 256, 0, stream>>>(reinterpret_cast<const float*>(in), ldi, reinterpret_cast<float*>(out), ldo, M, N, mode, a, b, row_scale);
  else if (in_fp32)
    glu_kernel<float, bf16><<<grid, 256, 0, stream>>>(reinterpret_cast<const float*>(in), ldi, reinterpret_cast<bf16*>(out), ldo, M, N, mode, a, b, row_scale);
  else if (out_fp32)
    glu_kernel<bf16, float><<<grid, 256, 0, stream>>>(reinterpret_cast<const bf16*>(in), ldi, reinterpret_cast<float*>(out), ldo, M, N, mode, a, b, row_scale);
  else
    glu_kernel<bf16, bf16><<<grid, 256, 0, stream>>>(reinterpret_cast<const bf16*>(in), ldi, reinterpret_cast<bf16*>(out), ldo, M, N, mode, a, b, row_scale);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_dyt_f32(const float* x, long long ldx, int M, int D, float alpha, const float* gain, const float* shift, void* out,
                          long long ldo, float alpha2, const float* gain2, const float* shift2, void* out2, long long ldo2, int out_fp32,
                          void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(x != nullptr && gain != nullptr && out != nullptr && M >= 0 && D > 0, "lp_dyt_f32: bad arguments");
  LP_REQUIRE(out2 == nullptr || gain2 != nullptr, "lp_dyt_f32: a second output without its gain");
  if (M == 0) return 0;
  // bf16 rows of four are 8 bytes: their bases need 8-byte alignment, which the 16-byte test covers
  const bool v4 = vec4_ok(D, {x, gain, gain2, out, out2}, {ldx, ldo, out2 != nullptr ? ldo2 : 0});
  const unsigned grid = (unsigned)(((long long)M * (v4 ? D / 4 : D) + 255) / 256);
  if (out_fp32 && v4)
    dyt_f32_kernel<float, 4><<<grid, 256, 0, stream>>>(x, ldx, M, D, alpha, gain, shift, reinterpret_cast<float*>(out), ldo, alpha2, gain2,
                                                       shift2, reinterpret_cast<float*>(out2), ldo2);
  else if (out_fp32)
    dyt_f32_kernel<float, 1><<<grid, 256, 0, stream>>>(x, ldx, M, D, alpha, gain, shift, reinterpret_cast<float*>(out), ldo, alpha2, gain2,
                                                       shift2, reinterpret_cast<float*>(out2), ldo2);
  else if (v4)
    dyt_f32_kernel<bf16, 4><<<grid, 256, 0, stream>>>(x, ldx, M, D, alpha, gain, shift, reinterpret_cast<bf16*>(out), ldo, alpha2, gain2,
                                                      shift2, reinterpret_cast<bf16*>(out2), ldo2);
  else
    dyt_f32_kernel<bf16, 1><<<grid, 256, 0, stream>>>(x, ldx, M, D, alpha, gain, shift, reinterpret_cast<bf16*>(out), ldo, alpha2, gain2,
                                                      shift2, reinterpret_cast<bf16*>(out2), ldo2);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_rmsnorm_gated_f32(const float* x, long long ldx, int M, int D, const float* gain, float eps, const float* gate,
                                    long long ldg, void* out, long long ldo, int out_fp32, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(x != nullptr && gate != nullptr && out != nullptr && M >= 0 && D > 0, "lp_rmsnorm_gated_f32: bad arguments");
  if (M == 0) return 0;
  const unsigned grid = (unsigned)((M + NORM32_WARPS - 1) / NORM32_WARPS);
  const bool v4 = vec4_ok(D, {x, gate, out}, {ldx, ldg, ldo});
  if (out_fp32 && v4)
    rmsnorm_gated_f32_kernel<float, 4><<<grid, NORM32_WARPS * 32, 0, stream>>>(x, ldx, M, D, gain, eps, gate, ldg, reinterpret_cast<float*>(out), ldo);
  else if (out_fp32)
    rmsnorm_gated_f32_kernel<float, 1><<<grid, NORM32_WARPS * 32, 0, stream>>>(x, ldx, M, D, gain, eps, gate, ldg, reinterpret_cast<float*>(out), ldo);
  else if (v4)
    rmsnorm_gated_f32_kernel<bf16, 4><<<grid, NORM32_WARPS * 32, 0, stream>>>(x, ldx, M, D, gain, eps, gate, ldg, reinterpret_cast<bf16*>(out), ldo);
  else
    rmsnorm_gated_f32_kernel<bf16, 1><<<grid, NORM32_WARPS * 32, 0, stream>>>(x, ldx, M, D, gain, eps, gate, ldg, reinterpret_cast<bf16*>(out), ldo);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_gated_axpy_f32(float* x, long long ldx, const float* y, long long ldy, const float* y_bias, const float* g, long long ldg,
                                 const float* g_bias, float mult, int M, int N, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(x != nullptr && y != nullptr && M >= 0 && N > 0, "lp_gated_axpy_f32: bad arguments");
  if (M == 0) return 0;
  if (vec4_ok(N, {x, y, g}, {ldx, ldy, g != nullptr ? ldg : 0}))
    gated_axpy_f32_kernel<4><<<(unsigned)(((long long)M * (N / 4) + 255) / 256), 256, 0, stream>>>(x, ldx, y, ldy, y_bias, g, ldg, g_bias, mult, M, N);
  else
    gated_axpy_f32_kernel<1><<<(unsigned)(((long long)M * N + 255) / 256), 256, 0, stream>>>(x, ldx, y, ldy, y_bias, g, ldg, g_bias, mult, M, N);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_depth_average_f32(const float* hist, long long layer_stride, long long ldh, const float* coef, int n, float* out,
                                    long long ldo, float* copy, long long ldc, int M, int N, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(hist != nullptr && coef != nullptr && out != nullptr && n > 0 && M >= 0 && N > 0, "lp_depth_average_f32: bad arguments");
  if (M == 0) return 0;
  if (vec4_ok(N, {hist, out, copy}, {layer_stride, ldh, ldo, copy != nullptr ? ldc : 0}))
    depth_average_f32_kernel<4><<<(unsigned)(((long long)M * (N / 4) + 255) / 256), 256, 0, stream>>>(hist, layer_stride, ldh, coef, n, out, ldo,
                                                                                                    copy, ldc, M, N);
  else
    depth_average_f32_kernel<1><<<(unsigned)(((long long)M * N + 255) / 256), 256, 0, stream>>>(hist, layer_stride, ldh, coef, n, out, ldo,
                                                                                              copy, ldc, M, N);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int lp_axpy_f32(float* y, long long ldy, const float* x, long long ldx, float alpha, int M, int N, void* stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LP_REQUIRE(y != nullptr && x != nullptr && M >= 0 && N > 0, "lp_axpy_f32: bad arguments");
  if (M == 0) return 0;
  axpy_f32_kernel<<<(unsigned)(((long long)M * N + 255) / 256), 256, 0, stream>>>(y, ldy, x, ldx, alpha, M, N);
  note_launch();
  LP_CHECK_CUDA(cudaGetLastError());
  return 0;
}
