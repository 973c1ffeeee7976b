// What the sublayers of a layer return joins the residual stream, and the next layer's norm is taken, in one pass:
//
//   x += scale * sum_t term_t;      optionally   out = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w + b
//
// A term is a float row times a factor, or such a row normed first over the whole width, factor * y / sqrt(mean(y^2) + eps) *
// norm_w, or the rows that a mixture of experts left in the order of its experts: factor * sum_c weights[m, c] *
// rows[row[m * top + c]], choices in their order (weights null: 1 each).  All arithmetic is 32-bit.  One block a token; a
// token's sums depend on nothing else in the batch.
#include <math.h>

#include "common.cuh"

#define BJ_THREADS 256
#define BJ_MAX_TERMS 4

struct BranchTerm {
  const float* y;              // [M, d], or with `row` the experts' rows [*, d]
  const float* norm_w;         // [d] or null
  float eps, factor;
  const int* row;              // [M * top] or null
  const float* weights;        // [M, top] or null
  int top;
};

struct BranchArgs {
  BranchTerm term[BJ_MAX_TERMS];
  int terms;
  float* x;                    // [M, d]
  float scale;
  const float *w, *b;          // the norm behind (null: none); b may be null
  float eps;
  int d;
};

template <int V> struct BjVec { float v[V]; };
template <int V>
__device__ __forceinline__ BjVec<V> bj_ld(const float* p) {
  BjVec<V> r;
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int V>
__device__ __forceinline__ void bj_st(float* p, const BjVec<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}

// the sums of N values over the block, the same order everywhere
template <int N>
__device__ __forceinline__ void bj_block_sum(float (&v)[N], float (*s_part)[BJ_THREADS / 32]) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = rl_warp_sum(v[i]);
  __syncthreads();                       // s_part may still be read from an earlier call
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) s_part[i][warp] = v[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < N; ++i) {
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < BJ_THREADS / 32; ++w) t += s_part[i][w];
    v[i] = t;
  }
}

// V: columns a thread takes at a time; MAXV > 0: the row stays in registers, at most MAXV such pieces a thread; 0: any width,
// the row waits in shared memory (every thread reads back what it wrote itself)
template <typename T, int V, int MAXV>
__global__ void __launch_bounds__(BJ_THREADS)
branch_join_kernel(const BranchArgs a, T* __restrict__ out) {
  extern __shared__ __align__(16) float s_x[];
  __shared__ float s_part[BJ_MAX_TERMS][BJ_THREADS / 32];
  rl_pdl_trigger();
  rl_pdl_wait();
  const int d = a.d;
  const size_t m = blockIdx.x;
  float inv[BJ_MAX_TERMS];
  bool normed = false;
#pragma unroll
  for (int t = 0; t < BJ_MAX_TERMS; ++t) {
    inv[t] = 0.f;
    if (t < a.terms && a.term[t].norm_w) {
      normed = true;
      const float* y = a.term[t].y + m * d;
      for (int i = V * threadIdx.x; i < d; i += V * BJ_THREADS) {
        const BjVec<V> f = bj_ld<V>(y + i);
#pragma unroll
        for (int k = 0; k < V; ++k) inv[t] = fmaf(f.v[k], f.v[k], inv[t]);
      }
    }
  }
  if (normed) {
    bj_block_sum<BJ_MAX_TERMS>(inv, s_part);
#pragma unroll
    for (int t = 0; t < BJ_MAX_TERMS; ++t)
      if (t < a.terms) inv[t] = a.term[t].factor / sqrtf(inv[t] / (float)d + a.term[t].eps);
  }
  float* x = a.x + m * d;
  BjVec<V> keep[MAXV > 0 ? MAXV : 1];
  float sum[1] = {0.f};
  auto joined = [&](int i) {             // columns i .. i + V - 1 of the new x
    BjVec<V> s;
#pragma unroll
    for (int k = 0; k < V; ++k) s.v[k] = 0.f;
#pragma unroll
    for (int t = 0; t < BJ_MAX_TERMS; ++t) {
      if (t >= a.terms) break;
      const BranchTerm& q = a.term[t];
      if (q.row) {
        BjVec<V> e;
#pragma unroll
        for (int k = 0; k < V; ++k) e.v[k] = 0.f;
        for (int c = 0; c < q.top; ++c) {
          const float w = q.weights ? q.weights[m * q.top + c] : 1.f;
          const BjVec<V> f = bj_ld<V>(q.y + (size_t)q.row[m * q.top + c] * d + i);
#pragma unroll
          for (int k = 0; k < V; ++k) e.v[k] = fmaf(w, f.v[k], e.v[k]);
        }
#pragma unroll
        for (int k = 0; k < V; ++k) s.v[k] = fmaf(q.factor, e.v[k], s.v[k]);
      } else {
        const BjVec<V> f = bj_ld<V>(q.y + m * d + i);
        if (q.norm_w) {
          const BjVec<V> w = bj_ld<V>(q.norm_w + i);
#pragma unroll
          for (int k = 0; k < V; ++k) s.v[k] = fmaf(f.v[k] * inv[t], w.v[k], s.v[k]);
        } else {
#pragma unroll
          for (int k = 0; k < V; ++k) s.v[k] = fmaf(q.factor, f.v[k], s.v[k]);
        }
      }
    }
    BjVec<V> n = bj_ld<V>(x + i);
#pragma unroll
    for (int k = 0; k < V; ++k) n.v[k] = fmaf(a.scale, s.v[k], n.v[k]);
    bj_st<V>(x + i, n);
    return n;
  };
  auto store = [&](int i, const BjVec<V>& c, float r) {      // c: deviations from the mean
    const BjVec<V> w = bj_ld<V>(a.w + i);
    BjVec<V> o;
#pragma unroll
    for (int k = 0; k < V; ++k) o.v[k] = c.v[k] * r * w.v[k];
    if (a.b) {
      const BjVec<V> b = bj_ld<V>(a.b + i);
#pragma unroll
      for (int k = 0; k < V; ++k) o.v[k] += b.v[k];
    }
    if constexpr (V == 4 && sizeof(T) == 2) {
      __nv_bfloat162 lo = __floats2bfloat162_rn(o.v[0], o.v[1]), hi = __floats2bfloat162_rn(o.v[2], o.v[3]);
      *reinterpret_cast<uint2*>(out + m * d + i) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) rl_st(out + m * d + i + k, o.v[k]);
    }
  };
  if constexpr (MAXV > 0) {
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
      const int i = V * (threadIdx.x + j * BJ_THREADS);
      if (i < d) {
        keep[j] = joined(i);
#pragma unroll
        for (int k = 0; k < V; ++k) sum[0] += keep[j].v[k];
      }
    }
    if (!a.w) return;
    bj_block_sum<1>(sum, s_part);
    const float mean = sum[0] / (float)d;
    sum[0] = 0.f;
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
      const int i = V * (threadIdx.x + j * BJ_THREADS);
      if (i < d) {
#pragma unroll
        for (int k = 0; k < V; ++k) { keep[j].v[k] -= mean; sum[0] = fmaf(keep[j].v[k], keep[j].v[k], sum[0]); }
      }
    }
    bj_block_sum<1>(sum, s_part);
    const float r = 1.0f / sqrtf(sum[0] / (float)d + a.eps);
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
      const int i = V * (threadIdx.x + j * BJ_THREADS);
      if (i < d) store(i, keep[j], r);
    }
  } else {
    for (int i = V * threadIdx.x; i < d; i += V * BJ_THREADS) {
      const BjVec<V> n = joined(i);
      if (a.w) {
        bj_st<V>(s_x + i, n);
#pragma unroll
        for (int k = 0; k < V; ++k) sum[0] += n.v[k];
      }
    }
    if (!a.w) return;
    bj_block_sum<1>(sum, s_part);
    const float mean = sum[0] / (float)d;
    sum[0] = 0.f;
    for (int i = V * threadIdx.x; i < d; i += V * BJ_THREADS) {
      BjVec<V> n = bj_ld<V>(s_x + i);
#pragma unroll
      for (int k = 0; k < V; ++k) { n.v[k] -= mean; sum[0] = fmaf(n.v[k], n.v[k], sum[0]); }
      bj_st<V>(s_x + i, n);
    }
    bj_block_sum<1>(sum, s_part);
    const float r = 1.0f / sqrtf(sum[0] / (float)d + a.eps);
    for (int i = V * threadIdx.x; i < d; i += V * BJ_THREADS) store(i, bj_ld<V>(s_x + i), r);
  }
}

template <typename T>
static int bj_launch(const BranchArgs& a, T* out, int num, cudaStream_t stream) {
  uintptr_t bits = (uintptr_t)a.x | (uintptr_t)a.w | (uintptr_t)a.b | (uintptr_t)out;
  for (int t = 0; t < a.terms; ++t) bits |= (uintptr_t)a.term[t].y | (uintptr_t)a.term[t].norm_w;
  const bool vec = a.d % 4 == 0 && (bits & 15) == 0;
  if (vec && a.d <= 4 * BJ_THREADS * 2) {
    rl_launch_pdl(branch_join_kernel<T, 4, 2>, dim3(num), dim3(BJ_THREADS), 0, stream, a, out);
  } else if (vec && a.d <= 4 * BJ_THREADS * 4) {
    rl_launch_pdl(branch_join_kernel<T, 4, 4>, dim3(num), dim3(BJ_THREADS), 0, stream, a, out);
  } else if (vec && a.d <= 4 * BJ_THREADS * 8) {
    rl_launch_pdl(branch_join_kernel<T, 4, 8>, dim3(num), dim3(BJ_THREADS), 0, stream, a, out);
  } else {
    const size_t smem = a.w ? (size_t)a.d * sizeof(float) : 0;
    RL_REQUIRE(smem <= 40 * 1024, "rl_branch_join: %d columns exceed the %d this kernel holds", a.d, 10 * 1024);
    rl_launch_pdl(branch_join_kernel<T, 1, 0>, dim3(num), dim3(BJ_THREADS), smem, stream, a, out);
  }
  return RL_OK;
}

// x [M, d] float takes scale * the sum of `terms` (at most 4) terms; term t: ys[t] float rows, norm_ws[t] [d] or null with
// epss[t], factors[t], rows[t] ([M * tops[t]] ints) or null, weights[t] ([M, tops[t]]) or null (all host arrays of device
// pointers or numbers).  norm_w (float [d], null: no norm behind), norm_b (float [d] or null), norm_eps, out [M, d] in out_dtype.
extern "C" int rl_branch_join(float* x, float scale, int terms, const void* const* ys, const void* const* norm_ws, const float* epss,
                              const float* factors, const void* const* rows, const void* const* weights, const int* tops,
                              const float* norm_w, const float* norm_b, float norm_eps, void* out, int out_dtype, int num_tokens, int hidden,
                              cudaStream_t stream) {
  RL_REQUIRE(num_tokens >= 0 && hidden > 0 && terms >= 1 && terms <= BJ_MAX_TERMS, "rl_branch_join: bad sizes, or %d terms outside [1, %d]", terms, BJ_MAX_TERMS);
  RL_REQUIRE((norm_w == nullptr) == (out == nullptr) && (norm_w != nullptr || norm_b == nullptr), "rl_branch_join: the norm's weight and its output come together");
  if (num_tokens == 0) return RL_OK;
  BranchArgs a = {};
  for (int t = 0; t < terms; ++t) {
    RL_REQUIRE(ys[t] != nullptr && !(rows[t] && norm_ws[t]) && (!rows[t] || tops[t] > 0), "rl_branch_join: term %d: no rows, experts' rows that are normed, or no top", t);
    a.term[t] = {(const float*)ys[t], (const float*)norm_ws[t], epss[t], factors[t], (const int*)rows[t], (const float*)weights[t], tops[t]};
  }
  a.terms = terms; a.x = x; a.scale = scale; a.w = norm_w; a.b = norm_b; a.eps = norm_eps; a.d = hidden;
  int rc = RL_OK;
  if (out == nullptr || out_dtype == RL_F32) rc = bj_launch<float>(a, (float*)out, num_tokens, stream);
  else if (out_dtype == RL_BF16) rc = bj_launch<__nv_bfloat16>(a, (__nv_bfloat16*)out, num_tokens, stream);
  else RL_REQUIRE(false, "rl_branch_join: unknown dtype %d", out_dtype);
  if (rc != RL_OK) return rc;
  RL_LAUNCH_CHECK("rl_branch_join");
  return RL_OK;
}
