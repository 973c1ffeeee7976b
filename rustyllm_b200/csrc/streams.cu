// A residual made of several streams: X [M, S, d] float, all 32-bit.  A sublayer reads a weighted sum of a token's
// streams, normed; what it returns is mixed back into all of them at once:
//
//   read   u = sum_s coef[s] X[s];    out = u / sqrt(mean(u^2) + eps) * w           (coef null: the plain sum)
//   join   X[t] <- sum_s mix[s][t] X[s] + to[t] * (channel_scale * y)               (all t from the old X)
//   open   X[s] <- x0 for every s
//
// One kernel does a join (or an open) and the read that follows it: between two sublayers a token's streams are
// read once and written once, and the next sublayer's normed input is made while they are in registers.  y comes
// as a float row, or as the rows that a mixture of experts left in the order of its experts (row[m * top + c] is
// where the token's choice c lies) with the router's weights: y = sum_c weights[m, c] * rows[row[m * top + c]],
// choices in their order.  One block a token; a token's sums depend on nothing else in the batch.
#include <math.h>

#include "common.cuh"

#define ST_THREADS 256
#define ST_MAX_STREAMS 32
#define ST_MAX_FIXED 8         // up to here the number of streams is a compile-time constant

enum { ST_OPEN = 0, ST_JOIN = 1, ST_READ = 2 };

struct StreamArgs {
  float* X;                    // [M, S, d]
  const float* x0;             // open: [M, d]
  const float* y;              // join: [M, d], or with `row` the experts' rows [*, d]
  float y_factor;              // a constant on a dense y
  const int* row;              // [M * top] or null
  const float* weights;        // [M, top]
  int top;
  const float* channel_scale;  // [d] or null
  const float* mix;            // [S, S], from-stream major
  const float* to;             // [S]
  const float* coef;           // [S] or null (ones)
  const float* norm_w;         // [d]; null: nothing is read out after a join or an open
  float eps;
  const int* rows;             // read: the tokens whose sums are wanted, or null (all)
  int d, S;
};

template <int V> struct StVec;
template <> struct StVec<4> { float v[4]; };
template <> struct StVec<1> { float v[1]; };
template <int V>
__device__ __forceinline__ StVec<V> st_ld(const float* p) {
  StVec<V> r;
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int V>
__device__ __forceinline__ void st_st(float* p, const StVec<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}

// SN > 0: the number of streams; SN <= 0: at most -SN of them, their number is a.S.  V: columns a thread takes at a time.
template <typename T, int SN, int MODE, int V>
__global__ void __launch_bounds__(ST_THREADS)
streams_kernel(const StreamArgs a, T* __restrict__ out) {
  constexpr int SM = SN > 0 ? SN : -SN;
  constexpr int UN = SM <= ST_MAX_FIXED ? SM : 1;    // how far the loops over streams are unrolled
  extern __shared__ __align__(16) float s_u[];       // [d]: the sum that is read
  __shared__ float s_mix[SM * SM], s_to[SM], s_coef[SM], s_part[ST_THREADS / 32];
  const int S = SN > 0 ? SN : a.S;
  const int d = a.d;
  rl_pdl_trigger();
  // the coefficients are the model's: no kernel of a step writes them
  if (MODE == ST_JOIN) {
    for (int i = threadIdx.x; i < S * S; i += ST_THREADS) s_mix[i] = a.mix[i];
    for (int i = threadIdx.x; i < S; i += ST_THREADS) s_to[i] = a.to[i];
  }
  for (int i = threadIdx.x; i < S; i += ST_THREADS) s_coef[i] = a.coef ? a.coef[i] : 1.f;
  __syncthreads();
  rl_pdl_wait();
  const size_t m = blockIdx.x;                       // the output row
  const size_t tok = MODE == ST_READ && a.rows ? (size_t)a.rows[m] : m;
  float* X = a.X + tok * S * d;
  float ss = 0.f;
  for (int i = V * threadIdx.x; i < d; i += V * ST_THREADS) {
    StVec<V> x[SM];
    if (MODE == ST_OPEN) {
      const StVec<V> e = st_ld<V>(a.x0 + tok * d + i);
#pragma unroll UN
      for (int s = 0; s < SM; ++s)
        if (s < S) { x[s] = e; st_st<V>(X + (size_t)s * d + i, e); }
    } else {
#pragma unroll UN
      for (int s = 0; s < SM; ++s)
        if (s < S) x[s] = st_ld<V>(X + (size_t)s * d + i);
    }
    StVec<V> u;
#pragma unroll
    for (int k = 0; k < V; ++k) u.v[k] = 0.f;
    if (MODE == ST_JOIN) {
      StVec<V> y;
      if (a.row) {
#pragma unroll
        for (int k = 0; k < V; ++k) y.v[k] = 0.f;
        for (int c = 0; c < a.top; ++c) {
          const float w = a.weights[tok * a.top + c];
          const StVec<V> r = st_ld<V>(a.y + (size_t)a.row[tok * a.top + c] * d + i);
#pragma unroll
          for (int k = 0; k < V; ++k) y.v[k] = fmaf(w, r.v[k], y.v[k]);
        }
      } else {
        y = st_ld<V>(a.y + tok * d + i);
#pragma unroll
        for (int k = 0; k < V; ++k) y.v[k] *= a.y_factor;
      }
      if (a.channel_scale) {
        const StVec<V> c = st_ld<V>(a.channel_scale + i);
#pragma unroll
        for (int k = 0; k < V; ++k) y.v[k] *= c.v[k];
      }
#pragma unroll UN
      for (int t = 0; t < SM; ++t)
        if (t < S) {
          StVec<V> n;
#pragma unroll
          for (int k = 0; k < V; ++k) n.v[k] = s_to[t] * y.v[k];
#pragma unroll UN
          for (int s = 0; s < SM; ++s)
            if (s < S) {
              const float c = s_mix[s * S + t];
#pragma unroll
              for (int k = 0; k < V; ++k) n.v[k] = fmaf(c, x[s].v[k], n.v[k]);
            }
          st_st<V>(X + (size_t)t * d + i, n);
#pragma unroll
          for (int k = 0; k < V; ++k) u.v[k] = fmaf(s_coef[t], n.v[k], u.v[k]);
        }
    } else {
#pragma unroll UN
      for (int s = 0; s < SM; ++s)
        if (s < S) {
#pragma unroll
          for (int k = 0; k < V; ++k) u.v[k] = fmaf(s_coef[s], x[s].v[k], u.v[k]);
        }
    }
    if (a.norm_w) {
#pragma unroll
      for (int k = 0; k < V; ++k) ss = fmaf(u.v[k], u.v[k], ss);
      st_st<V>(s_u + i, u);
    }
  }
  if (!a.norm_w) return;
  ss = rl_warp_sum(ss);
  if ((threadIdx.x & 31) == 0) s_part[threadIdx.x >> 5] = ss;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (int w = 0; w < ST_THREADS / 32; ++w) total += s_part[w];
  const float r = 1.0f / sqrtf(total / (float)d + a.eps);
  T* o = out + m * d;
  for (int i = V * threadIdx.x; i < d; i += V * ST_THREADS) {      // (every thread reads back what it wrote itself)
    const StVec<V> u = st_ld<V>(s_u + i), w = st_ld<V>(a.norm_w + i);
    if constexpr (V == 4 && sizeof(T) == 2) {
      __nv_bfloat162 lo = __floats2bfloat162_rn(u.v[0] * r * w.v[0], u.v[1] * r * w.v[1]);
      __nv_bfloat162 hi = __floats2bfloat162_rn(u.v[2] * r * w.v[2], u.v[3] * r * w.v[3]);
      *reinterpret_cast<uint2*>(o + i) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) rl_st(o + i + k, u.v[k] * r * w.v[k]);
    }
  }
}

template <typename T, int MODE>
static int st_launch(const StreamArgs& a, T* out, int num, cudaStream_t stream) {
  const size_t smem = a.norm_w ? (size_t)a.d * sizeof(float) : 0;
  RL_REQUIRE(smem <= 40 * 1024, "rl_streams: %d columns exceed the %d this kernel holds", a.d, 10 * 1024);
  const uintptr_t bits = (uintptr_t)a.X | (uintptr_t)a.x0 | (uintptr_t)a.y | (uintptr_t)a.channel_scale | (uintptr_t)a.norm_w | (uintptr_t)out;
  const bool vec = a.d % 4 == 0 && (bits & 15) == 0;
#define RL_ST(SN, V) rl_launch_pdl(streams_kernel<T, SN, MODE, V>, dim3(num), dim3(ST_THREADS), smem, stream, a, out)
  if (!vec || a.S > ST_MAX_FIXED) {
    if (a.S <= ST_MAX_FIXED) RL_ST(-ST_MAX_FIXED, 1);
    else RL_ST(-ST_MAX_STREAMS, 1);
    return RL_OK;
  }
  switch (a.S) {
    case 1: RL_ST(1, 4); break;
    case 2: RL_ST(2, 4); break;
    case 3: RL_ST(3, 4); break;
    case 4: RL_ST(4, 4); break;
    case 5: RL_ST(5, 4); break;
    case 6: RL_ST(6, 4); break;
    case 7: RL_ST(7, 4); break;
    default: RL_ST(8, 4); break;
  }
#undef RL_ST
  return RL_OK;
}

// mode 0 open, 1 join, 2 read (see above).  X [M, S, d] float; x0 [M, d] (open); y [M, d] float times y_factor, or with
// row ([M * top] ints) and weights ([M, top]) the experts' rows (join); channel_scale [d] or null; mix [S, S], to [S]
// (join); coef [S] or null; norm_w [d] and out [num, d] in out_dtype (both null after an open or a join: nothing is
// read out); rows [num] or null (read).  num = M, or the number of rows wanted.
extern "C" int rl_streams(int mode, float* X, const float* x0, const float* y, float y_factor, const int* row, const float* weights,
                          int top, const float* channel_scale, const float* mix, const float* to, const float* coef,
                          const float* norm_w, float eps, const int* rows, int num, int streams, int hidden, void* out, int out_dtype,
                          cudaStream_t stream) {
  RL_REQUIRE(num >= 0 && hidden > 0, "rl_streams: bad sizes M=%d d=%d", num, hidden);
  RL_REQUIRE(streams >= 1 && streams <= ST_MAX_STREAMS, "rl_streams: %d streams outside [1, %d]", streams, ST_MAX_STREAMS);
  RL_REQUIRE(mode >= 0 && mode <= 2 && X != nullptr, "rl_streams: unknown mode %d or no streams", mode);
  RL_REQUIRE(mode != ST_OPEN || x0 != nullptr, "rl_streams: opening needs the row to copy");
  RL_REQUIRE(mode != ST_JOIN || (y != nullptr && mix != nullptr && to != nullptr), "rl_streams: a join needs y, mix and to");
  RL_REQUIRE((row == nullptr) == (weights == nullptr) && (row == nullptr || top > 0), "rl_streams: experts' rows come with weights and top");
  RL_REQUIRE((norm_w == nullptr) == (out == nullptr), "rl_streams: the norm's weight and its output come together");
  RL_REQUIRE(mode != ST_READ || norm_w != nullptr, "rl_streams: a read without a norm writes nothing");
  if (num == 0) return RL_OK;
  StreamArgs a = {X, x0, y, y_factor, row, weights, top, channel_scale, mix, to, coef, norm_w, eps, rows, hidden, streams};
  int rc = RL_OK;
  if (out_dtype == RL_F32)
    rc = mode == ST_OPEN ? st_launch<float, ST_OPEN>(a, (float*)out, num, stream)
         : mode == ST_JOIN ? st_launch<float, ST_JOIN>(a, (float*)out, num, stream)
                           : st_launch<float, ST_READ>(a, (float*)out, num, stream);
  else if (out_dtype == RL_BF16)
    rc = mode == ST_OPEN ? st_launch<__nv_bfloat16, ST_OPEN>(a, (__nv_bfloat16*)out, num, stream)
         : mode == ST_JOIN ? st_launch<__nv_bfloat16, ST_JOIN>(a, (__nv_bfloat16*)out, num, stream)
                           : st_launch<__nv_bfloat16, ST_READ>(a, (__nv_bfloat16*)out, num, stream);
  else
    RL_REQUIRE(false, "rl_streams: unknown dtype %d", out_dtype);
  if (rc != RL_OK) return rc;
  RL_LAUNCH_CHECK("rl_streams");
  return RL_OK;
}
