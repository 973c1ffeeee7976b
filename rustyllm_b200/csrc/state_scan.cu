// Recurrences with a matrix state per head whose output reads the current token's write, carried from step to step:
//
//   gated linear attention   S_t = diag(a_t) S_{t-1} + k_t v_t^T,   o_t = S_t^T (q_scale q_t)          (S: dk x dv)
//                            a_t = sigmoid(z_t)^(1/tau), a decay a key channel and token, from the float z
//   gated delta rule         q, k divided by sqrt(sum of squares + unit_eps) a head, q times q_scale;
//                            g_t = exp(-exp(rate_h) softplus(a_t + dt_bias_h)),  beta_t = sigmoid(b_t), a number a head;
//                            S = g_t S_{t-1};  u = beta_t (v_t - S^T k_t);  S_t = S + k_t u^T;  o_t = S_t^T q_t
//                            (query/key heads may be shared: head h reads group h / hpg)
//
// All arithmetic behind the loads is 32-bit; the state is float [H, dv, dk] in the sequence's slot, as in linear_scan.cu.
//
// A block owns COLS columns of one head's state of one sequence and walks the sequence's tokens of the step in order.
// Eight neighbouring lanes share CPT columns, each with NPT of their rows in registers (two floats an instruction): a q, k or
// decay fetched from shared memory serves CPT columns, and a 16-byte load of a warp costs four passes however few addresses
// it has.  The walk depends on itself token after token, so everything that does not is taken off it: PW warps of their own
// keep the next two tiles of TILE tokens in flight as raw values, form decays, step sizes, unit vectors and the scalar k . q,
// and leave them in the other half of a double buffer, one barrier a tile; a tile's tokens beyond the sequence are staged so
// that they change nothing (k = q = 0, decays of 1), which leaves the walk without branches; and the lanes' parts of a
// tile's outputs are added behind the walk, scattered over the lanes while they are added (7 shuffles for 8 tokens of a
// column).  The delta rule reads both products with the old state in one pass: with a = S^T k and b = S^T q,
// u = beta (v - g a) and o = g b + (k . q) u, so only a's three shuffles stand in the chain from token to token.
// 2,048 tokens of 16 heads, 64 x 128 linear and 128 x 128 delta: 827 and 1,274 us with loads that were converted as they
// arrived, 229 and 356 us with raw values two tiles ahead; two columns a lane and 32 a block: 207 and 396 us, and at 32 heads
// 211 and 397 us instead of 280 and 516.
// Every sum's order is fixed by the sizes alone (both launch shapes add the eight lanes in the same order), so a position's
// output does not depend on how the sequence was cut into steps or on the batch.
#include <math.h>

#include "common.cuh"

#define SS_MAX_DK 256

enum { SS_LINEAR = 0, SS_DELTA = 1 };

template <typename T>
struct StateScanArgs {
  const T *q, *k, *v;
  int ldq, ldk, ldv;
  const float* z;                     // linear: [M, ldz], head h at columns [h * dk, (h + 1) * dk)
  int ldz;
  float inv_tau;
  const T *a_raw, *b_raw;             // delta: [M, lda], [M, ldb], a column a head
  int lda, ldb;
  const float *rate, *dt_bias;        // delta: [H]
  float unit_eps;
  float q_scale;
  const int *cu_seqlens, *seq_slots;
  float* state;
  long long state_stride;
  float* out;
  int ldo, H, hpg, dk, dv;
};

// two floats an instruction (packed fp32 of sm_100)
__device__ __forceinline__ float2 ss_fma2(float2 a, float2 b, float2 c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d)
      : "l"(*reinterpret_cast<uint64_t*>(&a)), "l"(*reinterpret_cast<uint64_t*>(&b)), "l"(*reinterpret_cast<uint64_t*>(&c)));
  return *reinterpret_cast<float2*>(&d);
}
__device__ __forceinline__ float2 ss_mul2(float2 a, float2 b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(*reinterpret_cast<uint64_t*>(&a)), "l"(*reinterpret_cast<uint64_t*>(&b)));
  return *reinterpret_cast<float2*>(&d);
}
__device__ __forceinline__ float ss_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// sigmoid(z)^(1/tau) = exp(-softplus(-z) / tau): with the accurate functions in a 32-bit run; in a bfloat16 run, whose z has
// 8 bits of its inputs behind it, with the fast exponential and logarithm (absolute error of the logarithm about 1e-7)
__device__ __forceinline__ float ss_decay(float z, float inv_tau, float) { return expf(-ss_softplus(-z) * inv_tau); }
__device__ __forceinline__ float ss_decay(float z, float inv_tau, __nv_bfloat16) {
  return __expf(-(fmaxf(-z, 0.f) + __logf(1.0f + __expf(-fabsf(z)))) * inv_tau);
}

template <typename T, int MODE, int NPT, int COLS, int CPT, int TILE, int PW>
__global__ void __launch_bounds__(8 * COLS / CPT + 32 * PW)
state_scan_kernel(const StateScanArgs<T> a) {
  constexpr bool DELTA = MODE == SS_DELTA;
  constexpr int R = 8, DKP = R * NPT, NE = DKP / 32, TPW = TILE / PW;
  constexpr int CONSUMERS = R * COLS / CPT;
  static_assert(TILE % PW == 0 && NPT % 4 == 0 && TILE <= R, "tile shapes");
  __shared__ __align__(16) float s_k[2][TILE][DKP], s_q[2][TILE][DKP];
  __shared__ __align__(16) float s_w[DELTA ? 1 : 2][DELTA ? 1 : TILE][DELTA ? 4 : DKP];
  __shared__ __align__(16) float s_v[2][TILE][COLS];
  __shared__ __align__(16) float4 s_c[2][TILE];            // delta: g, beta, k . q
  rl_pdl_trigger();
  rl_pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS;
  const int lo = a.cu_seqlens[b], hi = a.cu_seqlens[b + 1];
  const int tiles = (hi - lo + TILE - 1) / TILE;
  if (tiles <= 0) return;
  const int dk = a.dk, dv = a.dv;

  if (threadIdx.x >= CONSUMERS) {
    // ---------------- producers: a warp takes TPW tokens of every tile ----------------
    const int pw = (threadIdx.x - CONSUMERS) >> 5, lane = threadIdx.x & 31;
    const size_t qk0 = (size_t)(h / a.hpg) * dk;
    constexpr int VE = (TPW * COLS + 31) / 32;             // values a lane stages
    // what a lane fetches of a tile, as it lies in memory: nothing here waits for a load.  Every load is made, at the nearest
    // token and column there is; what does not belong to the tile is dropped when the tile is staged.
    struct Raw {
      T q[TPW][NE], k[TPW][NE], v[VE], a, b;
      float z[DELTA ? 1 : TPW][DELTA ? 1 : NE];
    };
    const float neg_rate = DELTA ? -expf(a.rate[h]) : 0.f, dt_bias = DELTA ? a.dt_bias[h] : 0.f;
    auto fetch = [&](Raw& f, int tile) {
      const int t0 = lo + tile * TILE + pw * TPW;
#pragma unroll
      for (int tt = 0; tt < TPW; ++tt) {
        const size_t t = min(t0 + tt, hi - 1);
#pragma unroll
        for (int e = 0; e < NE; ++e) {
          const int n = min(lane + 32 * e, dk - 1);
          f.q[tt][e] = a.q[t * a.ldq + qk0 + n];
          f.k[tt][e] = a.k[t * a.ldk + qk0 + n];
          if constexpr (!DELTA) f.z[tt][e] = a.z[t * a.ldz + (size_t)h * dk + n];
        }
      }
#pragma unroll
      for (int e = 0; e < VE; ++e) {
        const int idx = lane + 32 * e;
        f.v[e] = a.v[(size_t)min(t0 + min(idx / COLS, TPW - 1), hi - 1) * a.ldv + (size_t)h * dv + min(c0 + idx % COLS, dv - 1)];
      }
      if constexpr (DELTA) {
        const size_t t = min(t0 + min(lane, TPW - 1), hi - 1);
        f.a = a.a_raw[t * a.lda + h];
        f.b = a.b_raw[t * a.ldb + h];
      }
    };
    auto commit = [&](const Raw& f, int tile) {
      const int buf = tile & 1, t0 = lo + tile * TILE + pw * TPW;
      float q[TPW][NE], k[TPW][NE], rq[TPW], rk[TPW], kq[TPW];
#pragma unroll
      for (int tt = 0; tt < TPW; ++tt) {
        rq[tt] = a.q_scale; rk[tt] = 1.f; kq[tt] = 0.f;
#pragma unroll
        for (int e = 0; e < NE; ++e) {
          const bool in = t0 + tt < hi && lane + 32 * e < dk;
          q[tt][e] = in ? rl_ld(&f.q[tt][e]) : 0.f;
          k[tt][e] = in ? rl_ld(&f.k[tt][e]) : 0.f;
        }
      }
      if constexpr (DELTA) {
        float sq[TPW], sk[TPW];
#pragma unroll
        for (int tt = 0; tt < TPW; ++tt) {
          sq[tt] = sk[tt] = 0.f;
#pragma unroll
          for (int e = 0; e < NE; ++e) {
            sq[tt] = fmaf(q[tt][e], q[tt][e], sq[tt]);
            sk[tt] = fmaf(k[tt][e], k[tt][e], sk[tt]);
            kq[tt] = fmaf(k[tt][e], q[tt][e], kq[tt]);
          }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
          for (int tt = 0; tt < TPW; ++tt) {
            sq[tt] += __shfl_xor_sync(0xffffffffu, sq[tt], o);
            sk[tt] += __shfl_xor_sync(0xffffffffu, sk[tt], o);
            kq[tt] += __shfl_xor_sync(0xffffffffu, kq[tt], o);
          }
        }
#pragma unroll
        for (int tt = 0; tt < TPW; ++tt) {
          rq[tt] = a.q_scale / sqrtf(sq[tt] + a.unit_eps);
          rk[tt] = 1.0f / sqrtf(sk[tt] + a.unit_eps);
          kq[tt] *= rq[tt] * rk[tt];
        }
        if (lane < TPW) {
          const bool in = t0 + lane < hi;
          float mine = 0.f;
#pragma unroll
          for (int tt = 0; tt < TPW; ++tt) mine = lane == tt ? kq[tt] : mine;
          s_c[buf][pw * TPW + lane] = make_float4(in ? expf(neg_rate * ss_softplus(rl_ld(&f.a) + dt_bias)) : 1.f,
                                                  in ? 1.0f / (1.0f + expf(-rl_ld(&f.b))) : 0.f, mine, 0.f);
        }
      }
#pragma unroll
      for (int tt = 0; tt < TPW; ++tt) {
#pragma unroll
        for (int e = 0; e < NE; ++e) {
          const int n = lane + 32 * e;
          s_q[buf][pw * TPW + tt][n] = q[tt][e] * rq[tt];
          s_k[buf][pw * TPW + tt][n] = k[tt][e] * rk[tt];
          if constexpr (!DELTA)
            s_w[buf][pw * TPW + tt][n] = (t0 + tt < hi && n < dk) ? ss_decay(f.z[tt][e], a.inv_tau, T()) : 1.f;
        }
      }
#pragma unroll
      for (int e = 0; e < VE; ++e) {
        const int idx = lane + 32 * e, tt = idx / COLS;
        if (tt < TPW) s_v[buf][pw * TPW + tt][idx % COLS] = (t0 + tt < hi && c0 + idx % COLS < dv) ? rl_ld(&f.v[e]) : 0.f;
      }
    };
    if constexpr (TILE > 1) {
      Raw even, odd;                                        // two tiles in flight
      fetch(even, 0);
      fetch(odd, 1);
      for (int i = 0; i < tiles; i += 2) {
        commit(even, i);
        fetch(even, i + 2);
        __syncthreads();
        if (i + 1 < tiles) {
          commit(odd, i + 1);
          fetch(odd, i + 3);
          __syncthreads();
        }
      }
    } else {
      Raw f;
      fetch(f, 0);
      for (int i = 0; i < tiles; ++i) {
        commit(f, i);
        if (i + 1 < tiles) fetch(f, i + 1);
        __syncthreads();
      }
    }
    return;
  }

  // ---------------- the walk ----------------
  const int r = threadIdx.x % R, c = threadIdx.x / R * CPT;
  // row 4 R (i / 4) + 4 r + i % 4: a lane's rows in runs of four, neighbouring lanes side by side (whole lines of the state)
  auto row_of = [&](int i) { return 4 * R * (i / 4) + 4 * r + i % 4; };
  float* st = a.state + (size_t)a.seq_slots[b] * a.state_stride + ((size_t)h * dv + c0 + c) * dk;
  const bool vec = dk % 4 == 0;
  float2 S[CPT][NPT / 2];
#pragma unroll
  for (int j = 0; j < CPT; ++j) {
    const bool live = c0 + c + j < dv;
#pragma unroll
    for (int i = 0; i < NPT; i += 4) {
      const int row = row_of(i);
      if (vec) {
        const float4 f = (live && row < dk) ? *reinterpret_cast<const float4*>(st + (size_t)j * dk + row) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[j][i / 2] = make_float2(f.x, f.y);
        S[j][i / 2 + 1] = make_float2(f.z, f.w);
      } else {
        float f[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) f[u] = (live && row + u < dk) ? st[(size_t)j * dk + row + u] : 0.f;
        S[j][i / 2] = make_float2(f[0], f[1]);
        S[j][i / 2 + 1] = make_float2(f[2], f[3]);
      }
    }
  }
  for (int tile = 0; tile < tiles; ++tile) {
    const int buf = tile & 1;
    __syncthreads();
    float part[CPT][TILE];
#pragma unroll
    for (int tt = 0; tt < TILE; ++tt) {
      const float4* k4 = reinterpret_cast<const float4*>(&s_k[buf][tt][4 * r]);
      const float4* q4 = reinterpret_cast<const float4*>(&s_q[buf][tt][4 * r]);
      float v[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) v[j] = s_v[buf][tt][c + j];
      if constexpr (DELTA) {
        const float4 cc = s_c[buf][tt];
        float2 kk[NPT / 2], pa[CPT][2], pb[CPT][2];
#pragma unroll
        for (int j = 0; j < CPT; ++j) pa[j][0] = pa[j][1] = pb[j][0] = pb[j][1] = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < NPT / 4; ++i) {
          const float4 kf = k4[R * i], qf = q4[R * i];
          kk[2 * i] = make_float2(kf.x, kf.y);
          kk[2 * i + 1] = make_float2(kf.z, kf.w);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            pa[j][0] = ss_fma2(S[j][2 * i], kk[2 * i], pa[j][0]);
            pa[j][1] = ss_fma2(S[j][2 * i + 1], kk[2 * i + 1], pa[j][1]);
            pb[j][0] = ss_fma2(S[j][2 * i], make_float2(qf.x, qf.y), pb[j][0]);
            pb[j][1] = ss_fma2(S[j][2 * i + 1], make_float2(qf.z, qf.w), pb[j][1]);
          }
        }
        float sk[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) sk[j] = (pa[j][0].x + pa[j][0].y) + (pa[j][1].x + pa[j][1].y);
#pragma unroll
        for (int o = R / 2; o > 0; o >>= 1) {
#pragma unroll
          for (int j = 0; j < CPT; ++j) sk[j] += __shfl_xor_sync(0xffffffffu, sk[j], o);
        }
        const float2 g2 = make_float2(cc.x, cc.x);
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
#pragma unroll
          for (int i = 0; i < NPT / 2; ++i) S[j][i] = ss_mul2(S[j][i], g2);
        }
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          const float u = cc.y * fmaf(-cc.x, sk[j], v[j]);
          const float2 u2 = make_float2(u, u);
#pragma unroll
          for (int i = 0; i < NPT / 2; ++i) S[j][i] = ss_fma2(kk[i], u2, S[j][i]);
          const float sq = (pb[j][0].x + pb[j][0].y) + (pb[j][1].x + pb[j][1].y);
          part[j][tt] = fmaf(cc.x, sq, r == 0 ? u * cc.z : 0.f);
        }
      } else {
        const float4* w4 = reinterpret_cast<const float4*>(&s_w[buf][tt][4 * r]);
        float2 pb[CPT][2];
#pragma unroll
        for (int j = 0; j < CPT; ++j) pb[j][0] = pb[j][1] = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < NPT / 4; ++i) {
          const float4 kf = k4[R * i], qf = q4[R * i], wf = w4[R * i];
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            const float2 v2 = make_float2(v[j], v[j]);
            S[j][2 * i] = ss_fma2(make_float2(wf.x, wf.y), S[j][2 * i], ss_mul2(make_float2(kf.x, kf.y), v2));
            S[j][2 * i + 1] = ss_fma2(make_float2(wf.z, wf.w), S[j][2 * i + 1], ss_mul2(make_float2(kf.z, kf.w), v2));
            pb[j][0] = ss_fma2(S[j][2 * i], make_float2(qf.x, qf.y), pb[j][0]);
            pb[j][1] = ss_fma2(S[j][2 * i + 1], make_float2(qf.z, qf.w), pb[j][1]);
          }
        }
#pragma unroll
        for (int j = 0; j < CPT; ++j) part[j][tt] = (pb[j][0].x + pb[j][0].y) + (pb[j][1].x + pb[j][1].y);
      }
    }
    // the lanes' parts: halves of the tile's tokens change hands while they are added, until a lane holds one token
    int n = TILE;
#pragma unroll
    for (int o = R / 2; o > 0; o >>= 1) {
      if (n > 1) {
        n /= 2;
        const bool up = (r & o) != 0;
#pragma unroll
        for (int t = 0; t < TILE / 2; ++t) {
          if (t < n) {
#pragma unroll
            for (int j = 0; j < CPT; ++j) {
              const float send = up ? part[j][t] : part[j][t + n], keep = up ? part[j][t + n] : part[j][t];
              part[j][t] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
          }
        }
      } else {
#pragma unroll
        for (int j = 0; j < CPT; ++j) part[j][0] += __shfl_xor_sync(0xffffffffu, part[j][0], o);
      }
    }
    constexpr int LANES = R / TILE;                          // lanes that hold the same token
    const int t = lo + tile * TILE + r / LANES;
    if (r % LANES == 0 && t < hi) {
#pragma unroll
      for (int j = 0; j < CPT; ++j)
        if (c0 + c + j < dv) a.out[(size_t)t * a.ldo + (size_t)h * dv + c0 + c + j] = part[j][0];
    }
  }
#pragma unroll
  for (int j = 0; j < CPT; ++j) {
    if (c0 + c + j >= dv) break;
#pragma unroll
    for (int i = 0; i < NPT; i += 4) {
      const int row = row_of(i);
      float* p = st + (size_t)j * dk + row;
      if (vec) {
        if (row < dk) *reinterpret_cast<float4*>(p) = make_float4(S[j][i / 2].x, S[j][i / 2].y, S[j][i / 2 + 1].x, S[j][i / 2 + 1].y);
      } else {
        const float f[4] = {S[j][i / 2].x, S[j][i / 2].y, S[j][i / 2 + 1].x, S[j][i / 2 + 1].y};
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (row + u < dk) p[u] = f[u];
      }
    }
  }
}

template <typename T, int MODE>
static void ss_launch(const StateScanArgs<T>& a, int num_seqs, int wide, cudaStream_t stream) {
#define SS_GO(NPT, COLS, CPT, TILE, PW)                                                                                   \
  rl_launch_pdl(state_scan_kernel<T, MODE, NPT, COLS, CPT, TILE, PW>, dim3(num_seqs, a.H, (a.dv + COLS - 1) / COLS),      \
                dim3(8 * COLS / CPT + 32 * PW), 0, stream, a)
  if (wide) {                  // many tokens a sequence
    if (a.dk <= 32) SS_GO(4, 32, 2, 8, 4);
    else if (a.dk <= 64) SS_GO(8, 32, 2, 8, 4);
    else if (a.dk <= 128) SS_GO(16, 32, 2, 8, 4);
    else SS_GO(32, 16, 1, 4, 4);
  } else {                     // single tokens and short runs: the state's traffic is the work
    if (a.dk <= 32) SS_GO(4, 16, 1, 1, 1);
    else if (a.dk <= 64) SS_GO(8, 16, 1, 1, 1);
    else if (a.dk <= 128) SS_GO(16, 16, 1, 1, 1);
    else SS_GO(32, 16, 1, 1, 1);
  }
#undef SS_GO
}

static int ss_check(const char* who, int num_seqs, int num_heads, int dk, int dv, const float* state, long long state_stride) {
  RL_REQUIRE(num_seqs >= 0 && num_heads > 0 && num_heads <= 65535, "%s: bad sizes", who);
  RL_REQUIRE(dk > 0 && dk <= SS_MAX_DK && dv > 0, "%s: dk %d outside (0, %d] or dv %d", who, dk, SS_MAX_DK, dv);
  RL_REQUIRE(state != nullptr && state_stride >= (long long)num_heads * dk * dv && (dk % 4 != 0 || (((uintptr_t)state & 15) == 0 && state_stride % 4 == 0)),
             "%s: no state, rows too short, or rows of 16-byte pieces that are not 16-byte aligned", who);
  return RL_OK;
}

// Gated linear attention.  q, k [M, ld] with head h at columns [h * dk, (h + 1) * dk), v [M, ldv] with head h at [h * dv, ..),
// in `dtype`; z float [M, ldz]: the decay of key channel n of head h at token t is sigmoid(z[t, h * dk + n])^(1/tau).  state:
// float, this recurrence's [H, dv, dk] of slot s at state + s * state_stride.  out float [M, ldo].  wide != 0: the launch shape
// for many tokens a sequence; both shapes give the same bits.
extern "C" int rl_gated_linear_scan(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, int dtype, const float* z,
                                    int ldz, float tau, float q_scale, const int* cu_seqlens, const int* seq_slots, int num_seqs,
                                    float* state, long long state_stride, float* out, int ldo, int num_heads, int dk, int dv, int wide,
                                    cudaStream_t stream) {
  if (const int rc = ss_check("rl_gated_linear_scan", num_seqs, num_heads, dk, dv, state, state_stride)) return rc;
  RL_REQUIRE(z != nullptr && ldz >= num_heads * dk && tau > 0.f, "rl_gated_linear_scan: no decays, or tau %g not positive", (double)tau);
  if (num_seqs == 0) return RL_OK;
#define SS_ARGS(T)                                                                                                           \
  StateScanArgs<T> { (const T*)q, (const T*)k, (const T*)v, ldq, ldk, ldv, z, ldz, 1.0f / tau, nullptr, nullptr, 0, 0, nullptr, \
                     nullptr, 0.f, q_scale, cu_seqlens, seq_slots, state, state_stride, out, ldo, num_heads, 1, dk, dv }
  if (dtype == RL_F32) ss_launch<float, SS_LINEAR>(SS_ARGS(float), num_seqs, wide, stream);
  else if (dtype == RL_BF16) ss_launch<__nv_bfloat16, SS_LINEAR>(SS_ARGS(__nv_bfloat16), num_seqs, wide, stream);
  else RL_REQUIRE(false, "rl_gated_linear_scan: unknown dtype %d", dtype);
#undef SS_ARGS
  RL_LAUNCH_CHECK("rl_gated_linear_scan");
  return RL_OK;
}

// The gated delta rule.  q, k [M, ld] with group g at columns [g * dk, (g + 1) * dk) (head h reads group h / heads_per_group),
// v [M, ldv] with head h at [h * dv, ..); a_raw [M, lda], b_raw [M, ldb] with head h at column h: the decay is
// exp(-exp(rate[h]) softplus(a + dt_bias[h])), the step size sigmoid(b); all in `dtype`, rate and dt_bias float [H].
// State, output and `wide` as above.
extern "C" int rl_gated_delta_scan(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const void* a_raw, int lda,
                                   const void* b_raw, int ldb, int dtype, const float* rate, const float* dt_bias, float unit_eps,
                                   float q_scale, const int* cu_seqlens, const int* seq_slots, int num_seqs, float* state,
                                   long long state_stride, float* out, int ldo, int num_heads, int heads_per_group, int dk, int dv,
                                   int wide, cudaStream_t stream) {
  if (const int rc = ss_check("rl_gated_delta_scan", num_seqs, num_heads, dk, dv, state, state_stride)) return rc;
  RL_REQUIRE(heads_per_group > 0 && num_heads % heads_per_group == 0, "rl_gated_delta_scan: %d heads in groups of %d", num_heads, heads_per_group);
  RL_REQUIRE(a_raw != nullptr && b_raw != nullptr && rate != nullptr && dt_bias != nullptr && unit_eps > 0.f,
             "rl_gated_delta_scan: no decays or step sizes, or unit_eps %g not positive", (double)unit_eps);
  if (num_seqs == 0) return RL_OK;
#define SS_ARGS(T)                                                                                                           \
  StateScanArgs<T> { (const T*)q, (const T*)k, (const T*)v, ldq, ldk, ldv, nullptr, 0, 0.f, (const T*)a_raw, (const T*)b_raw, lda, \
                     ldb, rate, dt_bias, unit_eps, q_scale, cu_seqlens, seq_slots, state, state_stride, out, ldo, num_heads, heads_per_group, dk, dv }
  if (dtype == RL_F32) ss_launch<float, SS_DELTA>(SS_ARGS(float), num_seqs, wide, stream);
  else if (dtype == RL_BF16) ss_launch<__nv_bfloat16, SS_DELTA>(SS_ARGS(__nv_bfloat16), num_seqs, wide, stream);
  else RL_REQUIRE(false, "rl_gated_delta_scan: unknown dtype %d", dtype);
#undef SS_ARGS
  RL_LAUNCH_CHECK("rl_gated_delta_scan");
  return RL_OK;
}
