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
//                            A warp owns a channel (its row of either matrix) for 16 tokens whose inputs wait in
//                            shared memory; the lane that ends up with a token's sums advances its state.
// rl_short_conv_step         the causal filter in front, one token a sequence: filter and shift of the kept inputs
//                            in one kernel (a thread owns a channel of a sequence, so nobody else reads them).
#include <math.h>

#include "common.cuh"

#define GR_CH 16
#define GR_STEPS 8
#define GR_STEP_TOKENS 16

__device__ __forceinline__ float gr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gr_gelu(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// the token's step of the recurrence: S -> S + (h S + b); log a
struct GrStep { float log_a, h, b; };
__device__ __forceinline__ GrStep gr_step(float u, float zr, float zi, float rate_sp) {
  GrStep s;
  s.log_a = -rate_sp * gr_sigmoid(zr);
  s.h = expm1f(s.log_a);
  s.b = sqrtf(-s.h * (2.0f + s.h)) * gr_sigmoid(zi) * u;
  return s;
}
__device__ __forceinline__ float gr_advance(float S, float h, float b) { return S + fmaf(h, S, b); }

// u: channel c of token m at u[(c / part) * u_part + m * part + c % part]; z: float, its two sums at
// z[(c / part) * z_part + m * 2 part + c % part] (decay gate) and + part (input gate).
template <typename T, int TC>
__global__ void __launch_bounds__(GR_CH * TC)
gated_recurrence_kernel(const T* __restrict__ u, long long u_part, const float* __restrict__ z, long long z_part,
                        const float* __restrict__ z_bias, const float* __restrict__ lam, float rate, const T* __restrict__ y, int ldy,
                        T* __restrict__ out, int ldo, const int* __restrict__ cu_seqlens, const int* __restrict__ seq_slots,
                        float* __restrict__ state, long long state_stride, int W, int part) {
  __shared__ float s_h[TC][GR_CH], s_b[TC][GR_CH];
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
  float* st = state + (size_t)seq_slots[b] * state_stride;
  const T* up = u + (size_t)blk * u_part + at;
  const float* zp = z + (size_t)blk * z_part + at;
  float carry = live ? st[c] : 0.f;
  // a token's three inputs are requested one span ahead
  T ru[GR_STEPS], ry[GR_STEPS];
  float rr[GR_STEPS], ri[GR_STEPS];
  auto fetch = [&](int first) {
#pragma unroll
    for (int l = 0; l < GR_STEPS; ++l) {
      const int m = first + l;
      if (live && m < hi) {
        ru[l] = up[(size_t)m * part];
        rr[l] = zp[(size_t)m * 2 * part];
        ri[l] = zp[(size_t)m * 2 * part + part];
        ry[l] = y[(size_t)m * ldy + c];
      }
    }
  };
  fetch(lo + tc * GR_STEPS);
  for (int t0 = lo; t0 < hi; t0 += TC * GR_STEPS) {
    const int first = t0 + tc * GR_STEPS;
    float sh[GR_STEPS], sb[GR_STEPS], gy[GR_STEPS];
    float L = 0.f, B = 0.f;
#pragma unroll
    for (int l = 0; l < GR_STEPS; ++l) {
      sh[l] = 0.f; sb[l] = 0.f; gy[l] = 0.f;
      if (live && first + l < hi) {
        const GrStep s = gr_step(rl_ld(&ru[l]), rr[l] + br, ri[l] + bi, rate_sp);
        sh[l] = s.h; sb[l] = s.b;
        gy[l] = gr_gelu(rl_ld(&ry[l]));
        L += s.log_a;
        B = gr_advance(B, s.h, s.b);
      }
    }
    if (t0 + TC * GR_STEPS < hi) fetch(first + TC * GR_STEPS);
    __syncthreads();                       // the previous span's steps have been read
    s_h[tc][ch] = expm1f(L);
    s_b[tc][ch] = B;
    __syncthreads();
    float S = carry, mine = carry;
#pragma unroll
    for (int j = 0; j < TC; ++j) {
      if (j == tc) mine = S;
      S = gr_advance(S, s_h[j][ch], s_b[j][ch]);
    }
    carry = S;
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
    const GrStep s = gr_step(s_in[lane * part + n], mr + z_bias[(size_t)blk * 2 * part + n], mi + z_bias[(size_t)blk * 2 * part + part + n],
                             rate_sp);
    float* st = state + (size_t)seq_slots[m] * state_stride + c;
    const float S = gr_advance(*st, s.h, s.b);
    *st = S;
    rl_st(out + (size_t)m * ldo + c, S * gr_gelu(rl_ld(y + (size_t)m * ldy + c)));
  }
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
  const bool many = longest > 4 * GR_STEPS;
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
