// A linear recurrence with one state a channel, whose decay and input gate are functions of the channel's own
// (filtered) input:
//
//   r = sigmoid(zr + br),  i = sigmoid(zi + bi)          zr, zi: a square matrix a part of the channels, times u
//   log a = -rate * r * softplus(lam);   S_t = exp(log a) S_{t-1} + sqrt(1 - exp(2 log a)) * i * u_t
//   out_t = S_t * gelu_tanh(y_t)                         (y: the branch beside the recurrence, as projected)
//
// The state starts at zero and lives per slot as float [width].  Everything but the stored u, y and out is 32-bit.
// Where the decay is close to 1 (a memory of hundreds of tokens and more) exp(log a) has lost the digits that matter:
// rounded to float it is off by the same amount token after token.  So a step is held as h = exp(log a) - 1 (expm1):
// S + (h S + b), with 1 - a^2 = -h (2 + h), and a span of steps as expm1 of the sum of their logarithms.
//
// rl_gated_recurrence        prompts and portions: the gates' products zr, zi are given (a matrix product a part of
//                            the channels).  A block owns GR_CH channels of one sequence and walks its tokens in
//                            spans of TC * GR_STEPS: a thread takes GR_STEPS consecutive tokens of one channel,
//                            reduces them to one step of the same form, the threads' steps are composed in order
//                            through shared memory, and each replays its tokens from its own start.
// rl_gated_recurrence_step   one token a sequence: the gates' products, the recurrence and the output in one kernel.
//                            bfloat16: a block takes 16 channels (32 matrix rows) for up to 64 tokens on the tensor
//                            cores.  Any shape: a warp owns a channel for 16 tokens whose inputs wait in shared
//                            memory; the lane that ends up with a token's sums advances its state.
// rl_short_conv_step         the causal filter in front, one token a sequence: filter and shift of the kept inputs
//                            in one kernel (a thread owns a channel of a sequence, so nobody else reads them).
#include <math.h>

#include "common.cuh"
#include "small_product.cuh"

#define GR_CH 16
#define GR_STEPS 4
#define GR_STEP_TOKENS 16

__device__ __forceinline__ float gr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gr_gelu(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// the token's step of the recurrence: S -> S + (h S + b); log a
struct GrStep { float log_a, h, b; };
// A 32-bit run takes the accurate functions; a bfloat16 run (whose inputs carry 8 bits and whose kernel would be bound by
// instructions) the fast exponential, division and reciprocal square root, and e^x - 1 near 0 by the first terms of its
// power series: all of them float and good to about 2^-20.
template <typename T> struct GrMath;
template <> struct GrMath<float> {
  static __device__ __forceinline__ float sigmoid(float z) { return gr_sigmoid(z); }
  static __device__ __forceinline__ float expm1(float x) { return expm1f(x); }
  static __device__ __forceinline__ float root(float x) { return sqrtf(x); }
  static __device__ __forceinline__ float gelu(float z) { return gr_gelu(z); }
};
template <> struct GrMath<__nv_bfloat16> {
  static __device__ __forceinline__ float sigmoid(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
  static __device__ __forceinline__ float expm1(float x) {      // x <= 0; the series' next term is below 2^-20 of x up to |x| = 1/4
    const float near0 = x * fmaf(x, fmaf(x, fmaf(x, fmaf(x, 1.0f / 120.0f, 1.0f / 24.0f), 1.0f / 6.0f), 0.5f), 1.0f);
    return x > -0.25f ? near0 : __expf(x) - 1.0f;
  }
  static __device__ __forceinline__ float root(float x) { return x * rsqrtf(fmaxf(x, 1e-37f)); }
  static __device__ __forceinline__ float gelu(float z) {       // z / (1 + e^{-2y}), y the argument of the tanh
    const float y = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return __fdividef(z, 1.0f + __expf(fminf(-2.0f * y, 80.0f)));
  }
};
template <typename T>
__device__ __forceinline__ GrStep gr_step(float u, float zr, float zi, float rate_sp) {
  GrStep s;
  s.log_a = -rate_sp * GrMath<T>::sigmoid(zr);
  s.h = GrMath<T>::expm1(s.log_a);
  s.b = GrMath<T>::root(-s.h * (2.0f + s.h)) * GrMath<T>::sigmoid(zi) * u;
  return s;
}
__device__ __forceinline__ float gr_advance(float S, float h, float b) { return S + fmaf(h, S, b); }

// u: channel c of token m at u[(c / part) * u_part + m * part + c % part]; z: float, its two sums at
// z[(c / part) * z_part + m * 2 part + c % part] (decay gate) and + part (input gate).
template <typename T, int TC>
__global__ void __launch_bounds__(GR_CH * TC, TC > 8 ? 2 : 1)
gated_recurrence_kernel(const T* __restrict__ u, long long u_part, const float* __restrict__ z, long long z_part,
                        const float* __restrict__ z_bias, const float* __restrict__ lam, float rate, const T* __restrict__ y, int ldy,
                        T* __restrict__ out, int ldo, const int* __restrict__ cu_seqlens, const int* __restrict__ seq_slots,
                        float* __restrict__ state, long long state_stride, int W, int part) {
  static_assert(GR_CH == 16, "a warp holds two runs of tokens of the same channels");
  __shared__ float s_h[2][TC / 2][GR_CH], s_b[2][TC / 2][GR_CH];      // a pair of runs as one step; two spans in turn
  rl_pdl_trigger();
  const int ch = threadIdx.x % GR_CH, tc = threadIdx.x / GR_CH;
  const int c = blockIdx.x * GR_CH + ch;
  const bool live = c < W;
  const int blk = live ? c / part : 0, at = live ? c - blk * part : 0;
  const float rate_sp = live ? rate * gr_softplus(lam[c]) : 0.f;
  const float br = live ? z_bias[(size_t)blk * 2 * part + at] : 0.f, bi = live ? z_bias[(size_t)blk * 2 * part + part + at] : 0.f;
  rl_pdl_wait();
  const int b = blockIdx.y;
  const int lo = cu_seqlens[b], hi = cu_seqlens[b + 1];
  if (lo >= hi) return;
  float* st = state + (size_t)seq_slots[b] * state_stride;
  const T* up = u + (size_t)blk * u_part + at;
  const float* zp = z + (size_t)blk * z_part + at;
  const T* yp = y + (live ? c : 0);
  float carry = live ? st[c] : 0.f;
  // a token's three inputs are requested one span ahead
  T ru[GR_STEPS], ry[GR_STEPS];
  float rr[GR_STEPS], ri[GR_STEPS];
  auto fetch = [&](int first) {
#pragma unroll
    for (int l = 0; l < GR_STEPS; ++l) {
      const int m = min(first + l, hi - 1);          // (a row behind the last one is loaded and not used)
      ru[l] = up[(size_t)m * part];
      rr[l] = zp[(size_t)m * 2 * part];
      ri[l] = zp[(size_t)m * 2 * part + part];
      ry[l] = yp[(size_t)m * ldy];
    }
  };
  fetch(lo + tc * GR_STEPS);
  int buf = 0;
  for (int t0 = lo; t0 < hi; t0 += TC * GR_STEPS, buf ^= 1) {
    const int first = t0 + tc * GR_STEPS;
    float sh[GR_STEPS], sb[GR_STEPS], gy[GR_STEPS];
    float L = 0.f, B = 0.f;
#pragma unroll
    for (int l = 0; l < GR_STEPS; ++l) {
      const bool valid = first + l < hi;             // no branch: the steps' long chains overlap
      const GrStep s = gr_step<T>(rl_ld(&ru[l]), rr[l] + br, ri[l] + bi, rate_sp);
      sh[l] = valid ? s.h : 0.f;
      sb[l] = valid ? s.b : 0.f;
      gy[l] = GrMath<T>::gelu(rl_ld(&ry[l]));
      L += valid ? s.log_a : 0.f;
      B = gr_advance(B, sh[l], sb[l]);
    }
    if (t0 + TC * GR_STEPS < hi) fetch(first + TC * GR_STEPS);
    // the two runs of a warp joined, then the pairs in order.  (A buffer is written again two spans later; the barrier of
    // the span between has seen every reader leave.)
    const float h = GrMath<T>::expm1(L);
    const float oL = __shfl_xor_sync(0xffffffffu, L, GR_CH), oh = __shfl_xor_sync(0xffffffffu, h, GR_CH);
    const float oB = __shfl_xor_sync(0xffffffffu, B, GR_CH);
    if (tc & 1) {
      s_h[buf][tc >> 1][ch] = GrMath<T>::expm1(L + oL);
      s_b[buf][tc >> 1][ch] = gr_advance(oB, h, B);
    }
    __syncthreads();
    float S = carry, mine = carry;
#pragma unroll
    for (int j = 0; j < TC / 2; ++j) {
      if (j == tc >> 1) mine = S;
      S = gr_advance(S, s_h[buf][j][ch], s_b[buf][j][ch]);
    }
    carry = S;
    if (tc & 1) mine = gr_advance(mine, oh, oB);
#pragma unroll
    for (int l = 0; l < GR_STEPS; ++l) {
      mine = gr_advance(mine, sh[l], sb[l]);
      if (live && first + l < hi) rl_st(out + (size_t)(first + l) * ldo + c, mine * gy[l]);
    }
  }
  if (live && tc == 0) st[c] = carry;
}

// Eight consecutive weights, bf16 or float, as floats.
__device__ __forceinline__ void gr_ld8(const __nv_bfloat16* p, float (&w)[8]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
  for (int k = 0; k < 4; ++k) { const float2 f = __bfloat1622float2(h[k]); w[2 * k] = f.x; w[2 * k + 1] = f.y; }
}
__device__ __forceinline__ void gr_ld8(const float* p, float (&w)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  w[0] = a.x; w[1] = a.y; w[2] = a.z; w[3] = a.w; w[4] = b.x; w[5] = b.y; w[6] = b.z; w[7] = b.w;
}

// grid (ceil(part / 8), parts, token groups); 8 warps, a channel each.  u [M, W]: token m's row; w [parts, 2 part, part].
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
gated_recurrence_step_kernel(const T* __restrict__ u, int ldu, const T* __restrict__ w, const float* __restrict__ z_bias,
                             const float* __restrict__ lam, float rate, const T* __restrict__ y, int ldy, T* __restrict__ out,
                             int ldo, const int* __restrict__ seq_slots, float* __restrict__ state, long long state_stride, int M,
                             int part) {
  extern __shared__ __align__(16) float s_in[];      // [GR_STEP_TOKENS][part]
  rl_pdl_trigger();
  const int blk = blockIdx.y, m0 = blockIdx.z * GR_STEP_TOKENS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = blockIdx.x * 8 + warp;
  const T* wr = w + ((size_t)blk * 2 * part + n) * part;
  const T* wi = wr + (size_t)part * part;
  const int toks = min(GR_STEP_TOKENS, M - m0);
  // the first weights are requested before the wait: no kernel of a step writes them
  float a[8], g[8];
  if (VEC && n < part && 8 * lane < part) { gr_ld8(wr + 8 * lane, a); gr_ld8(wi + 8 * lane, g); }
  rl_pdl_wait();
  for (int i = threadIdx.x; i < GR_STEP_TOKENS * part; i += 256) {
    const int m = i / part, k = i - m * part;
    s_in[i] = m < toks ? rl_ld(u + (size_t)(m0 + m) * ldu + (size_t)blk * part + k) : 0.f;
  }
  __syncthreads();
  if (n >= part) return;
  float zr[GR_STEP_TOKENS], zi[GR_STEP_TOKENS];
#pragma unroll
  for (int m = 0; m < GR_STEP_TOKENS; ++m) zr[m] = zi[m] = 0.f;
  if (VEC) {
    for (int k = 8 * lane; k < part; k += 256) {
      if (k >= 256) { gr_ld8(wr + k, a); gr_ld8(wi + k, g); }
#pragma unroll
      for (int m = 0; m < GR_STEP_TOKENS; ++m) {
        if (m < toks) {
          const float4 x0 = *reinterpret_cast<const float4*>(s_in + m * part + k);
          const float4 x1 = *reinterpret_cast<const float4*>(s_in + m * part + k + 4);
          const float xs[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
          for (int e = 0; e < 8; ++e) { zr[m] = fmaf(a[e], xs[e], zr[m]); zi[m] = fmaf(g[e], xs[e], zi[m]); }
        }
      }
    }
  } else {
    for (int k = lane; k < part; k += 32) {
      const float av = rl_ld(wr + k), gv = rl_ld(wi + k);
#pragma unroll
      for (int m = 0; m < GR_STEP_TOKENS; ++m) {
        const float xv = s_in[m * part + k];
        zr[m] = fmaf(av, xv, zr[m]);
        zi[m] = fmaf(gv, xv, zi[m]);
      }
    }
  }
  float mr = 0.f, mi = 0.f;
#pragma unroll
  for (int m = 0; m < GR_STEP_TOKENS; ++m) {
    if (m < toks) {
      const float vr = rl_warp_sum(zr[m]), vi = rl_warp_sum(zi[m]);
      if (lane == m) { mr = vr; mi = vi; }
    }
  }
  if (lane < toks) {
    const int c = blk * part + n;
    const int m = m0 + lane;
    const float rate_sp = rate * gr_softplus(lam[c]);
    const GrStep s = gr_step<T>(s_in[lane * part + n], mr + z_bias[(size_t)blk * 2 * part + n], mi + z_bias[(size_t)blk * 2 * part + part + n],
                             rate_sp);
    float* st = state + (size_t)seq_slots[m] * state_stride + c;
    const float S = gr_advance(*st, s.h, s.b);
    *st = S;
    rl_st(out + (size_t)m * ldo + c, S * GrMath<T>::gelu(rl_ld(y + (size_t)m * ldy + c)));
  }
}

#define GR_MMA_CH (SP_ROWS / 2)
template <int TW>
__global__ void __launch_bounds__(SP_THREADS)
gated_recurrence_step_mma_kernel(const __nv_bfloat16* __restrict__ u, int ldu, const __nv_bfloat16* __restrict__ w,
                                 const float* __restrict__ z_bias, const float* __restrict__ lam, float rate,
                                 const __nv_bfloat16* __restrict__ y, int ldy, __nv_bfloat16* __restrict__ out, int ldo,
                                 const int* __restrict__ seq_slots, float* __restrict__ state, long long state_stride, int M, int part) {
  extern __shared__ __align__(128) uint8_t gr_smem[];
  rl_pdl_trigger();
  const SpLayout L = sp_layout(part, TW);
  const int blk = blockIdx.y, n0 = blockIdx.x * GR_MMA_CH, m0 = blockIdx.z * 16 * TW;
  const int chans = min(GR_MMA_CH, part - n0), toks = min(16 * TW, M - m0);
  // rows 0 .. 15: the channels' decay-gate rows, 16 .. 31: their input-gate rows (a row beyond the part repeats a live one)
  const __nv_bfloat16* wb = w + (size_t)blk * 2 * part * part;
  sp_fetch(gr_smem, 0, SP_ROWS, SP_ROWS, part, L, [&](int r) {
    const int ch = min(r % GR_MMA_CH, chans - 1);
    return wb + (size_t)((r / GR_MMA_CH) * part + n0 + ch) * part;
  });
  const int ch = threadIdx.x % GR_MMA_CH;
  const bool live = ch < chans;
  const int c = blk * part + n0 + (live ? ch : 0);
  const float rate_sp = rate * gr_softplus(lam[c]);
  const float br = z_bias[(size_t)blk * 2 * part + n0 + (live ? ch : 0)];
  const float bi = z_bias[(size_t)blk * 2 * part + part + n0 + (live ? ch : 0)];
  rl_pdl_wait();
  sp_fetch(gr_smem, L.x_off, 16 * TW, toks, part, L, [&](int r) { return u + (size_t)(m0 + r) * ldu + (size_t)blk * part; });
  sp_commit();
  // what the epilogue needs besides the sums, requested beside the operands
  constexpr int PER = 16 * TW * GR_MMA_CH / SP_THREADS;      // (token, channel) pairs a thread
  float S[PER], yv[PER];
  float* st[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int m = threadIdx.x / GR_MMA_CH + i * (SP_THREADS / GR_MMA_CH);
    S[i] = yv[i] = 0.f;
    st[i] = nullptr;
    if (live && m < toks) {
      st[i] = state + (size_t)seq_slots[m0 + m] * state_stride + c;
      S[i] = *st[i];
      yv[i] = __bfloat162float(y[(size_t)(m0 + m) * ldy + c]);
    }
  }
  sp_wait_all();
  __syncthreads();
  sp_multiply<TW>(gr_smem, L);
  const __nv_bfloat16* s_u = reinterpret_cast<const __nv_bfloat16*>(gr_smem + L.x_off);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int m = threadIdx.x / GR_MMA_CH + i * (SP_THREADS / GR_MMA_CH);
    if (st[i] == nullptr) continue;
    const GrStep s = gr_step<__nv_bfloat16>(__bfloat162float(s_u[m * L.ld + n0 + ch]), sp_sum<TW>(gr_smem, L, ch, m) + br,
                                            sp_sum<TW>(gr_smem, L, GR_MMA_CH + ch, m) + bi, rate_sp);
    const float next = gr_advance(S[i], s.h, s.b);
    *st[i] = next;
    out[(size_t)(m0 + m) * ldo + c] = __float2bfloat16_rn(next * GrMath<__nv_bfloat16>::gelu(yv[i]));
  }
}

template <int TW>
static int gr_step_mma(const void* u, int ldu, const void* w, const float* z_bias, const float* lam, float rate, const void* y, int ldy,
                       void* out, int ldo, const int* seq_slots, int num_seqs, float* state, long long state_stride, int width, int part,
                       cudaStream_t stream) {
  const SpLayout L = sp_layout(part, TW);
  static int reserved = 48 * 1024;
  if ((int)L.bytes > reserved) {
    cudaError_t e = cudaFuncSetAttribute(gated_recurrence_step_mma_kernel<TW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)L.bytes);
    RL_REQUIRE(e == cudaSuccess, "rl_gated_recurrence_step: cannot reserve %u bytes of shared memory: %s", L.bytes, cudaGetErrorString(e));
    reserved = (int)L.bytes;
  }
  const dim3 grid((part + GR_MMA_CH - 1) / GR_MMA_CH, width / part, (num_seqs + 16 * TW - 1) / (16 * TW));
  rl_launch_pdl(gated_recurrence_step_mma_kernel<TW>, grid, dim3(SP_THREADS), L.bytes, stream, (const __nv_bfloat16*)u, ldu,
                (const __nv_bfloat16*)w, z_bias, lam, rate, (const __nv_bfloat16*)y, ldy, (__nv_bfloat16*)out, ldo, seq_slots, state,
                state_stride, num_seqs, part);
  RL_LAUNCH_CHECK("rl_gated_recurrence_step");
  return RL_OK;
}

// state: kept inputs float [taps - 1, C] a slot, oldest first (as rl_short_conv).  A fresh slot's are zero.
template <typename T>
__global__ void __launch_bounds__(128)
short_conv_step_kernel(const T* __restrict__ u, int ldu, const float* __restrict__ w, const float* __restrict__ bias, int act, int C,
                       int taps, const int* __restrict__ seq_slots, float* __restrict__ state, long long state_stride,
                       T* __restrict__ out, int ldo) {
  rl_pdl_trigger();
  const int m = blockIdx.y, c = blockIdx.x * 128 + threadIdx.x;
  const bool live = c < C;
  const float b0 = live && bias ? bias[c] : 0.f;
  rl_pdl_wait();
  if (!live) return;
  float* st = state + (size_t)seq_slots[m] * state_stride + c;
  float acc = b0;
  float kept[8];
  const float cur = rl_ld(u + (size_t)m * ldu + c);
#pragma unroll
  for (int j = 0; j < 8; ++j)
    if (j < taps - 1) kept[j] = st[(size_t)j * C];
#pragma unroll
  for (int j = 0; j < 8; ++j)
    if (j < taps - 1) acc = fmaf(w[(size_t)c * taps + j], kept[j], acc);
  acc = fmaf(w[(size_t)c * taps + taps - 1], cur, acc);
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    if (j + 1 < taps - 1) st[(size_t)j * C] = kept[j + 1];
    else if (j + 1 == taps - 1) st[(size_t)j * C] = cur;
  }
  if (act == 1) acc = acc / (1.0f + expf(-acc));
  rl_st(out + (size_t)m * ldo + c, acc);
}

// One token a sequence, row m of u belonging to slot seq_slots[m].
extern "C" int rl_short_conv_step(const void* u, int ldu, int dtype, const float* w, const float* bias, int act, int channels, int taps,
                                  const int* seq_slots, int num_seqs, float* state, long long state_stride, void* out, int ldo,
                                  cudaStream_t stream) {
  RL_REQUIRE(num_seqs >= 0 && num_seqs <= 65535 && channels > 0, "rl_short_conv_step: bad sizes");
  RL_REQUIRE(taps >= 1 && taps <= 8, "rl_short_conv_step: %d taps outside [1, 8]", taps);
  RL_REQUIRE(ldu >= channels && ldo >= channels && (act == 0 || act == 1), "rl_short_conv_step: row strides too small or unknown activation");
  if (num_seqs == 0) return RL_OK;
  const dim3 grid((channels + 127) / 128, num_seqs);
  if (dtype == RL_F32)
    rl_launch_pdl(short_conv_step_kernel<float>, grid, dim3(128), 0, stream, (const float*)u, ldu, w, bias, act, channels, taps, seq_slots,
                  state, state_stride, (float*)out, ldo);
  else if (dtype == RL_BF16)
    rl_launch_pdl(short_conv_step_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, (const __nv_bfloat16*)u, ldu, w, bias, act, channels,
                  taps, seq_slots, state, state_stride, (__nv_bfloat16*)out, ldo);
  else
    RL_REQUIRE(false, "rl_short_conv_step: unknown dtype %d", dtype);
  RL_LAUNCH_CHECK("rl_short_conv_step");
  return RL_OK;
}

// u: part b of the channels at u + b * u_part, [M, part]; z float: at z + b * z_part, [M, 2 part] (decay gate's sums,
// then the input gate's, without bias); z_bias float [parts, 2 part]; lam float [width]; y, out [M, width] with row
// strides; state float [slots, state_stride] (this recurrence's [width] at the given pointer).
extern "C" int rl_gated_recurrence(const void* u, long long u_part, const float* z, long long z_part, const float* z_bias,
                                   const float* lam, float rate, const void* y, int ldy, void* out, int ldo, int dtype,
                                   const int* cu_seqlens, const int* seq_slots, int num_seqs, int longest, float* state,
                                   long long state_stride, int width, int part, cudaStream_t stream) {
  RL_REQUIRE(num_seqs >= 0 && num_seqs <= 65535 && width > 0 && part > 0 && width % part == 0, "rl_gated_recurrence: bad sizes (width %d in parts of %d)",
             width, part);
  RL_REQUIRE(ldy >= width && ldo >= width, "rl_gated_recurrence: row strides too small");
  if (num_seqs == 0) return RL_OK;
  const dim3 grid((width + GR_CH - 1) / GR_CH, num_seqs);
#define RL_GR(T, TC)                                                                                                              \
  rl_launch_pdl(gated_recurrence_kernel<T, TC>, grid, dim3(GR_CH * TC), 0, stream, (const T*)u, u_part, z, z_part, z_bias, lam, rate, \
                (const T*)y, ldy, (T*)out, ldo, cu_seqlens, seq_slots, state, state_stride, width, part)
  const bool many = longest > 8 * GR_STEPS;
  if (dtype == RL_F32) {
    if (many) RL_GR(float, 32); else RL_GR(float, 4);
  } else if (dtype == RL_BF16) {
    if (many) RL_GR(__nv_bfloat16, 32); else RL_GR(__nv_bfloat16, 4);
  } else {
    RL_REQUIRE(false, "rl_gated_recurrence: unknown dtype %d", dtype);
  }
#undef RL_GR
  RL_LAUNCH_CHECK("rl_gated_recurrence");
  return RL_OK;
}

// Channels a part that rl_gated_recurrence_step takes.
extern "C" int rl_gated_recurrence_step_max_part() { return 48 * 1024 / (GR_STEP_TOKENS * 4); }

// One token a sequence, row m belonging to slot seq_slots[m].  w [parts, 2 part, part] in dtype: a part's decay-gate
// matrix, then its input-gate matrix.  The rest as above.
extern "C" int rl_gated_recurrence_step(const void* u, int ldu, const void* w, const float* z_bias, const float* lam, float rate,
                                        const void* y, int ldy, void* out, int ldo, int dtype, const int* seq_slots, int num_seqs,
                                        float* state, long long state_stride, int width, int part, cudaStream_t stream) {
  RL_REQUIRE(num_seqs >= 0 && width > 0 && part > 0 && width % part == 0 && width / part <= 65535,
             "rl_gated_recurrence_step: bad sizes (width %d in parts of %d)", width, part);
  RL_REQUIRE(part <= rl_gated_recurrence_step_max_part(), "rl_gated_recurrence_step: parts of %d channels exceed the %d this kernel holds", part,
             rl_gated_recurrence_step_max_part());
  RL_REQUIRE(ldu >= width && ldy >= width && ldo >= width, "rl_gated_recurrence_step: row strides too small");
  if (num_seqs == 0) return RL_OK;
  if (dtype == RL_BF16 && part % 8 == 0 && ldu % 8 == 0 && (((uintptr_t)u | (uintptr_t)w) & 15) == 0 && num_seqs <= 65535 * 16 &&
      sp_layout(part, sp_token_warps(num_seqs)).bytes <= 200u * 1024u) {
#define RL_GM(TW) gr_step_mma<TW>(u, ldu, w, z_bias, lam, rate, y, ldy, out, ldo, seq_slots, num_seqs, state, state_stride, width, part, stream)
    switch (sp_token_warps(num_seqs)) {
      case 1: return RL_GM(1);
      case 2: return RL_GM(2);
      default: return RL_GM(4);
    }
#undef RL_GM
  }
  const dim3 grid((part + 7) / 8, width / part, (num_seqs + GR_STEP_TOKENS - 1) / GR_STEP_TOKENS);
  RL_REQUIRE(grid.z <= 65535, "rl_gated_recurrence_step: too many sequences (%d)", num_seqs);
  const size_t smem = (size_t)GR_STEP_TOKENS * part * sizeof(float);
  const bool vec = part % 8 == 0 && ((uintptr_t)w & 15) == 0;
#define RL_GS(T, V)                                                                                                                 \
  rl_launch_pdl(gated_recurrence_step_kernel<T, V>, grid, dim3(256), smem, stream, (const T*)u, ldu, (const T*)w, z_bias, lam, rate, \
                (const T*)y, ldy, (T*)out, ldo, seq_slots, state, state_stride, num_seqs, part)
  if (dtype == RL_F32) {
    if (vec) RL_GS(float, true); else RL_GS(float, false);
  } else if (dtype == RL_BF16) {
    if (vec) RL_GS(__nv_bfloat16, true); else RL_GS(__nv_bfloat16, false);
  } else {
    RL_REQUIRE(false, "rl_gated_recurrence_step: unknown dtype %d", dtype);
  }
#undef RL_GS
  RL_LAUNCH_CHECK("rl_gated_recurrence_step");
  return RL_OK;
}
