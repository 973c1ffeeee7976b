// Embedding gather, RMSNorm, SwiGLU and dtype conversion.
//
// Math in 32-bit throughout; storage of inputs/outputs is float or bf16 as the
// dtype tags say.  The residual stream these kernels read and write is always
// float.
//
// Formulas (SimonWaldherr/RustyLLM):
//   embedding : x = E[token, :]                         src/model.rs:7193
//   rms_norm  : y_i = x_i * 1/sqrt(sum(x^2)/n + eps) * w_i   src/model.rs:5429-5437
//   swiglu    : h_i = g_i / (1 + exp(-g_i)) * u_i       src/simd.rs:2403-2408
#include "common.cuh"

// ------------------------------------------------------------------ embedding
template <typename T>
__global__ void embedding_kernel(const T* __restrict__ table, const int* __restrict__ ids,
                                 float* __restrict__ out, int d, int vocab, int* __restrict__ err) {
  rl_pdl_trigger();
  rl_pdl_wait();
  const int m = blockIdx.x;
  int id = ids[m];
  if (id < 0 || id >= vocab) {  // refuse instead of reading outside the table
    if (threadIdx.x == 0) atomicExch(err, 1);
    id = 0;
  }
  const T* row = table + (size_t)id * d;
  float* o = out + (size_t)m * d;
  for (int i = threadIdx.x; i < d; i += blockDim.x) o[i] = rl_ld(row + i);
}

// err: optional device int, set to 1 when a token id lies outside [0, vocab).
extern "C" int rl_embedding(const void* table, int table_dtype, const int* ids, float* out,
                            int num_tokens, int hidden, int vocab, int* err, cudaStream_t stream) {
  RL_REQUIRE(num_tokens >= 0 && hidden > 0 && vocab > 0, "rl_embedding: bad sizes M=%d d=%d V=%d",
             num_tokens, hidden, vocab);
  RL_REQUIRE(err != nullptr, "rl_embedding: the error flag pointer is null");
  if (num_tokens == 0) return RL_OK;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == RL_F32)
    rl_launch_pdl(embedding_kernel<float>, num_tokens, threads, 0, stream, (const float*)table, ids, out, hidden, vocab, err);
  else if (table_dtype == RL_BF16)
    rl_launch_pdl(embedding_kernel<__nv_bfloat16>, num_tokens, threads, 0, stream, (const __nv_bfloat16*)table, ids, out, hidden, vocab, err);
  else
    RL_REQUIRE(false, "rl_embedding: unknown table dtype %d", table_dtype);
  RL_LAUNCH_CHECK("rl_embedding");
  return RL_OK;
}

// ------------------------------------------------------------------ RMSNorm
// One block per output row.  The sum of squares is taken in a fixed order that
// depends only on the row length and the block size, never on the batch.
template <typename TO, int THREADS>
__global__ void rmsnorm_kernel(const float* __restrict__ x, const float* __restrict__ w,
                               TO* __restrict__ out, const int* __restrict__ rows, int d, float eps) {
  rl_pdl_trigger();
  rl_pdl_wait();
  const int r = blockIdx.x;
  const float* xr = x + (size_t)(rows ? rows[r] : r) * d;
  float ss = 0.f;
  for (int i = threadIdx.x; i < d; i += THREADS) {
    const float v = xr[i];
    ss = fmaf(v, v, ss);
  }
  __shared__ float part[THREADS / 32];
  __shared__ float total;
  ss = rl_warp_sum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  if (threadIdx.x == 0) {
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; ++i) t += part[i];
    total = 1.0f / sqrtf(t / (float)d + eps);
  }
  __syncthreads();
  const float s = total;
  TO* o = out + (size_t)r * d;
  for (int i = threadIdx.x; i < d; i += THREADS) rl_st(o + i, xr[i] * s * w[i]);
}

// Rows of up to THREADS * 4 * MAXV floats, a multiple of 4 long, 16-byte aligned: the row
// stays in registers between the sum and the scaling, 16-byte loads, 8- or 16-byte stores.
template <typename TO, int THREADS, int MAXV>
__global__ void __launch_bounds__(THREADS)
rmsnorm_vec_kernel(const float* __restrict__ x, const float* __restrict__ w, TO* __restrict__ out,
                   const int* __restrict__ rows, int d, float eps) {
  rl_pdl_trigger();
  rl_pdl_wait();
  const int r = blockIdx.x;
  const float4* xr = reinterpret_cast<const float4*>(x + (size_t)(rows ? rows[r] : r) * d);
  const int nv = d / 4;
  float4 v[MAXV];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < MAXV; ++k) {
    const int i = threadIdx.x + k * THREADS;
    v[k] = i < nv ? xr[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    ss = fmaf(v[k].x, v[k].x, ss); ss = fmaf(v[k].y, v[k].y, ss);
    ss = fmaf(v[k].z, v[k].z, ss); ss = fmaf(v[k].w, v[k].w, ss);
  }
  __shared__ float part[THREADS / 32];
  __shared__ float total;
  ss = rl_warp_sum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  if (threadIdx.x == 0) {
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; ++i) t += part[i];
    total = 1.0f / sqrtf(t / (float)d + eps);
  }
  __syncthreads();
  const float s = total;
  const float4* w4 = reinterpret_cast<const float4*>(w);
  TO* o = out + (size_t)r * d;
#pragma unroll
  for (int k = 0; k < MAXV; ++k) {
    const int i = threadIdx.x + k * THREADS;
    if (i < nv) {
      const float4 g = w4[i];
      const float a = v[k].x * s * g.x, b = v[k].y * s * g.y, c = v[k].z * s * g.z, e = v[k].w * s * g.w;
      if constexpr (sizeof(TO) == 2) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, e);
        *reinterpret_cast<uint2*>(o + 4 * i) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
      } else {
        *reinterpret_cast<float4*>(o + 4 * i) = make_float4(a, b, c, e);
      }
    }
  }
}

// out[r, :] = rms_norm(x[rows ? rows[r] : r, :]) * w, for r in [0, num_rows).
extern "C" int rl_rmsnorm(const float* x, const float* weight, void* out, int out_dtype,
                          const int* rows, int num_rows, int hidden, float eps, cudaStream_t stream) {
  RL_REQUIRE(num_rows >= 0 && hidden > 0, "rl_rmsnorm: bad sizes rows=%d d=%d", num_rows, hidden);
  RL_REQUIRE(eps > 0.f, "rl_rmsnorm: eps must be > 0, got %g", (double)eps);
  if (num_rows == 0) return RL_OK;
  const bool vec = hidden % 4 == 0 && hidden <= 256 * 4 * 8 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)weight & 15) == 0 &&
                   ((uintptr_t)out & 15) == 0;
  if (vec && out_dtype == RL_BF16 && hidden <= 256 * 4 * 4)
    rl_launch_pdl(rmsnorm_vec_kernel<__nv_bfloat16, 256, 4>, num_rows, 256, 0, stream, x, weight, (__nv_bfloat16*)out, rows, hidden, eps);
  else if (vec && out_dtype == RL_BF16)
    rl_launch_pdl(rmsnorm_vec_kernel<__nv_bfloat16, 256, 8>, num_rows, 256, 0, stream, x, weight, (__nv_bfloat16*)out, rows, hidden, eps);
  else if (vec && out_dtype == RL_F32)
    rl_launch_pdl(rmsnorm_vec_kernel<float, 256, 8>, num_rows, 256, 0, stream, x, weight, (float*)out, rows, hidden, eps);
  else if (out_dtype == RL_F32)
    rl_launch_pdl(rmsnorm_kernel<float, 256>, num_rows, 256, 0, stream, x, weight, (float*)out, rows, hidden, eps);
  else if (out_dtype == RL_BF16)
    rl_launch_pdl(rmsnorm_kernel<__nv_bfloat16, 256>, num_rows, 256, 0, stream, x, weight, (__nv_bfloat16*)out, rows, hidden, eps);
  else
    RL_REQUIRE(false, "rl_rmsnorm: unknown output dtype %d", out_dtype);
  RL_LAUNCH_CHECK("rl_rmsnorm");
  return RL_OK;
}

// ------------------------------------------------------------------ SwiGLU
// gate_up: [M, 2*I] with the gate in columns [0, I) and up in [I, 2I); or, interleaved,
// gate_i in column 2i and up_i in column 2i + 1.
template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gu, T* __restrict__ out, int M, int I, int interleaved) {
  rl_pdl_trigger();
  rl_pdl_wait();
  const size_t total = (size_t)M * I;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (size_t)gridDim.x * blockDim.x) {
    const size_t m = idx / I;
    const int i = (int)(idx - m * I);
    const float g = rl_ld(gu + m * 2 * I + (interleaved ? 2 * i : i));
    const float u = rl_ld(gu + m * 2 * I + (interleaved ? 2 * i + 1 : I + i));
    rl_st(out + idx, g / (1.0f + expf(-g)) * u);
  }
}

// bf16, I a multiple of 8, 16-byte aligned rows: eight elements a thread
__global__ void swiglu_bf16x8_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ out, int M, int I) {
  rl_pdl_trigger();
  rl_pdl_wait();
  const int per_row = I / 8;
  const size_t total = (size_t)M * per_row;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
    const size_t m = idx / per_row;
    const int c = (int)(idx - m * per_row) * 8;
    const uint4 g4 = *reinterpret_cast<const uint4*>(gu + m * 2 * I + c);
    const uint4 u4 = *reinterpret_cast<const uint4*>(gu + m * 2 * I + I + c);
    const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&g4);
    const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&u4);
    uint4 o4;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o4);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 g = __bfloat1622float2(g2[k]), u = __bfloat1622float2(u2[k]);
      o2[k] = __floats2bfloat162_rn(g.x / (1.0f + expf(-g.x)) * u.x, g.y / (1.0f + expf(-g.y)) * u.y);
    }
    *reinterpret_cast<uint4*>(out + m * I + c) = o4;
  }
}

// bf16, interleaved (gate_i, up_i) pairs: four pairs in, four results out a thread
__global__ void swiglu_bf16_interleaved_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ out, size_t quads) {
  rl_pdl_trigger();
  rl_pdl_wait();
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < quads; idx += (size_t)gridDim.x * blockDim.x) {
    const uint4 v = *reinterpret_cast<const uint4*>(gu + idx * 8);
    const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&v);
    float r[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 gu2 = __bfloat1622float2(p[k]);
      r[k] = gu2.x / (1.0f + expf(-gu2.x)) * gu2.y;
    }
    __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
    *reinterpret_cast<uint2*>(out + idx * 4) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
  }
}

extern "C" int rl_swiglu(const void* gate_up, void* out, int dtype, int num_tokens,
                         int intermediate, int interleaved, cudaStream_t stream) {
  RL_REQUIRE(num_tokens >= 0 && intermediate > 0, "rl_swiglu: bad sizes M=%d I=%d", num_tokens, intermediate);
  if (num_tokens == 0) return RL_OK;
  const size_t total = (size_t)num_tokens * intermediate;
  const int threads = 256;
  const int blocks = (int)((total + threads - 1) / threads < rl_num_sms() * 16 ? (total + threads - 1) / threads : rl_num_sms() * 16);
  if (dtype == RL_BF16 && interleaved && intermediate % 4 == 0 && ((uintptr_t)gate_up & 15) == 0 && ((uintptr_t)out & 7) == 0) {
    const size_t quads = total / 4;      // rows are contiguous: [M, 2I] in, [M, I] out
    const int qblocks = (int)((quads + threads - 1) / threads < rl_num_sms() * 16 ? (quads + threads - 1) / threads : rl_num_sms() * 16);
    rl_launch_pdl(swiglu_bf16_interleaved_kernel, qblocks, threads, 0, stream, (const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, quads);
  } else if (dtype == RL_BF16 && !interleaved && intermediate % 8 == 0 && ((uintptr_t)gate_up & 15) == 0 && ((uintptr_t)out & 15) == 0) {
    const size_t vec = total / 8;
    const int vblocks = (int)((vec + threads - 1) / threads < rl_num_sms() * 16 ? (vec + threads - 1) / threads : rl_num_sms() * 16);
    rl_launch_pdl(swiglu_bf16x8_kernel, vblocks, threads, 0, stream, (const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, num_tokens, intermediate);
  } else if (dtype == RL_F32)
    rl_launch_pdl(swiglu_kernel<float>, blocks, threads, 0, stream, (const float*)gate_up, (float*)out, num_tokens, intermediate, interleaved);
  else if (dtype == RL_BF16)
    rl_launch_pdl(swiglu_kernel<__nv_bfloat16>, blocks, threads, 0, stream, (const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, num_tokens, intermediate, interleaved);
  else
    RL_REQUIRE(false, "rl_swiglu: unknown dtype %d", dtype);
  RL_LAUNCH_CHECK("rl_swiglu");
  return RL_OK;
}

// ------------------------------------------------------------------ dtype conversion
template <typename TI, typename TO>
__global__ void convert_kernel(const TI* __restrict__ in, TO* __restrict__ out, size_t n) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    rl_st(out + i, rl_ld(in + i));
}

extern "C" int rl_convert(const void* in, int in_dtype, void* out, int out_dtype, long long n,
                          cudaStream_t stream) {
  RL_REQUIRE(n >= 0, "rl_convert: negative length");
  if (n == 0) return RL_OK;
  const int threads = 256;
  const long long want = (n + threads - 1) / threads;
  const int blocks = (int)(want < rl_num_sms() * 16 ? want : rl_num_sms() * 16);
  if (in_dtype == RL_F32 && out_dtype == RL_BF16)
    convert_kernel<<<blocks, threads, 0, stream>>>((const float*)in, (__nv_bfloat16*)out, (size_t)n);
  else if (in_dtype == RL_BF16 && out_dtype == RL_F32)
    convert_kernel<<<blocks, threads, 0, stream>>>((const __nv_bfloat16*)in, (float*)out, (size_t)n);
  else
    RL_REQUIRE(false, "rl_convert: unsupported conversion %d -> %d", in_dtype, out_dtype);
  RL_LAUNCH_CHECK("rl_convert");
  return RL_OK;
}

// ------------------------------------------------------------------ embedding with learned positions
// x[m, :] = E[token_m, :] + P[position_m, :], summed in 32-bit (a learned absolute position
// table beside the token table; neither is scaled).
template <typename T>
__global__ void embedding_pos_kernel(const T* __restrict__ table, const T* __restrict__ pos_table,
                                     const int* __restrict__ ids, const int* __restrict__ positions,
                                     float* __restrict__ out, int d, int vocab, int max_pos, int* __restrict__ err) {
  rl_pdl_trigger();
  rl_pdl_wait();
  const int m = blockIdx.x;
  int id = ids[m], p = positions[m];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) atomicExch(err, 1);
    id = 0;
  }
  if (p < 0 || p >= max_pos) {     // a position beyond the table: refuse instead of reading outside it
    if (threadIdx.x == 0) atomicExch(err, 2);
    p = 0;
  }
  const T* row = table + (size_t)id * d;
  const T* prow = pos_table + (size_t)p * d;
  float* o = out + (size_t)m * d;
  for (int i = threadIdx.x; i < d; i += blockDim.x) o[i] = rl_ld(row + i) + rl_ld(prow + i);
}

extern "C" int rl_embedding_pos(const void* table, const void* pos_table, int table_dtype, const int* ids,
                                const int* positions, float* out, int num_tokens, int hidden, int vocab,
                                int max_positions, int* err, cudaStream_t stream) {
  RL_REQUIRE(num_tokens >= 0 && hidden > 0 && vocab > 0 && max_positions > 0,
             "rl_embedding_pos: bad sizes M=%d d=%d V=%d P=%d", num_tokens, hidden, vocab, max_positions);
  RL_REQUIRE(err != nullptr, "rl_embedding_pos: the error flag pointer is null");
  if (num_tokens == 0) return RL_OK;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == RL_F32)
    rl_launch_pdl(embedding_pos_kernel<float>, num_tokens, threads, 0, stream, (const float*)table, (const float*)pos_table,
                  ids, positions, out, hidden, vocab, max_positions, err);
  else if (table_dtype == RL_BF16)
    rl_launch_pdl(embedding_pos_kernel<__nv_bfloat16>, num_tokens, threads, 0, stream, (const __nv_bfloat16*)table,
                  (const __nv_bfloat16*)pos_table, ids, positions, out, hidden, vocab, max_positions, err);
  else
    RL_REQUIRE(false, "rl_embedding_pos: unknown table dtype %d", table_dtype);
  RL_LAUNCH_CHECK("rl_embedding_pos");
  return RL_OK;
}

// ------------------------------------------------------------------ scaled embedding with a hashed pair table
// x[m, :] = E[token_m, :] * scale + P[row_m, :], in 32-bit.  row_m = (prev_m * mul_prev + token_m * mul_cur) mod buckets,
// where prev_m is the token in front of token m in its sequence; a sequence's first token takes row `buckets` (the
// table has buckets + 1 rows).  The token in front of a step's first token of a sequence is per-slot state (an
// int32 a slot): the block of that first token reads it and then leaves the sequence's last token of this step
// there - it is the only block that touches the slot's entry, so nothing races.  pair_table null: the scaled
// embedding alone (the state is still kept).
template <typename T>
__global__ void embedding_pair_kernel(const T* __restrict__ table, const T* __restrict__ pair_table, const int* __restrict__ ids,
                                      const int* __restrict__ positions, const int* __restrict__ slot_of_token,
                                      const int* __restrict__ cu_seqlens, int num_seqs, int* __restrict__ last_token,
                                      long long state_stride, float scale, long long mul_prev, long long mul_cur, int buckets,
                                      float* __restrict__ out, int d, int vocab, int* __restrict__ err) {
  rl_pdl_trigger();
  rl_pdl_wait();
  __shared__ int s_prev;
  const int m = blockIdx.x;
  int id = ids[m];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) atomicExch(err, 1);
    id = 0;
  }
  if (threadIdx.x == 0) {
    const int slot = slot_of_token[m];
    const bool first_of_step = m == 0 || slot_of_token[m - 1] != slot;
    int prev = -1;
    if (!first_of_step) {
      prev = ids[m - 1];
    } else {
      int* st = last_token + (size_t)slot * state_stride;
      if (positions[m] > 0) prev = *st;
      int lo = 0, hi = num_seqs;            // the sequence b with cu_seqlens[b] <= m < cu_seqlens[b + 1]
      while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (cu_seqlens[mid] <= m) lo = mid; else hi = mid;
      }
      *st = ids[cu_seqlens[lo + 1] - 1];
    }
    if (prev >= vocab) prev = 0;            // a bad id was reported where it was read as a token
    s_prev = prev;
  }
  __syncthreads();
  const int prev = s_prev;
  const T* row = table + (size_t)id * d;
  float* o = out + (size_t)m * d;
  if (pair_table) {
    const long long r = prev < 0 ? (long long)buckets : ((long long)prev * mul_prev + (long long)id * mul_cur) % buckets;
    const T* prow = pair_table + (size_t)r * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) o[i] = fmaf(rl_ld(row + i), scale, rl_ld(prow + i));
  } else {
    for (int i = threadIdx.x; i < d; i += blockDim.x) o[i] = rl_ld(row + i) * scale;
  }
}

// last_token: int32, one entry a slot, `state_stride` ints apart.  mul_prev, mul_cur >= 0, buckets > 0 with a pair table.
extern "C" int rl_embedding_pair(const void* table, const void* pair_table, int table_dtype, const int* ids, const int* positions,
                                 const int* slot_of_token, const int* cu_seqlens, int num_seqs, int* last_token,
                                 long long state_stride, float scale, long long mul_prev, long long mul_cur, int buckets,
                                 float* out, int num_tokens, int hidden, int vocab, int* err, cudaStream_t stream) {
  RL_REQUIRE(num_tokens >= 0 && hidden > 0 && vocab > 0 && num_seqs >= 0, "rl_embedding_pair: bad sizes M=%d d=%d V=%d B=%d",
             num_tokens, hidden, vocab, num_seqs);
  RL_REQUIRE(err != nullptr && last_token != nullptr, "rl_embedding_pair: the error flag or the state pointer is null");
  RL_REQUIRE(pair_table == nullptr || (buckets > 0 && mul_prev >= 0 && mul_cur >= 0), "rl_embedding_pair: bad hash constants");
  if (num_tokens == 0) return RL_OK;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == RL_F32)
    rl_launch_pdl(embedding_pair_kernel<float>, num_tokens, threads, 0, stream, (const float*)table, (const float*)pair_table, ids,
                  positions, slot_of_token, cu_seqlens, num_seqs, last_token, state_stride, scale, mul_prev, mul_cur, buckets, out,
                  hidden, vocab, err);
  else if (table_dtype == RL_BF16)
    rl_launch_pdl(embedding_pair_kernel<__nv_bfloat16>, num_tokens, threads, 0, stream, (const __nv_bfloat16*)table,
                  (const __nv_bfloat16*)pair_table, ids, positions, slot_of_token, cu_seqlens, num_seqs, last_token, state_stride,
                  scale, mul_prev, mul_cur, buckets, out, hidden, vocab, err);
  else
    RL_REQUIRE(false, "rl_embedding_pair: unknown table dtype %d", table_dtype);
  RL_LAUNCH_CHECK("rl_embedding_pair");
  return RL_OK;
}

// ------------------------------------------------------------------ gelu, tanh form
// out = 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), in 32-bit, rounded once at the store.
template <typename T>
__global__ void gelu_tanh_kernel(const T* __restrict__ in, T* __restrict__ out, size_t total) {
  rl_pdl_trigger();
  rl_pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const float z = rl_ld(in + i);
    rl_st(out + i, 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))));
  }
}

extern "C" int rl_gelu_tanh(const void* in, void* out, int dtype, long long total, cudaStream_t stream) {
  RL_REQUIRE(total >= 0, "rl_gelu_tanh: negative size");
  if (total == 0) return RL_OK;
  const int threads = 256;
  const int blocks = (int)((total + threads - 1) / threads < 148 * 16 ? (total + threads - 1) / threads : 148 * 16);
  if (dtype == RL_F32)
    rl_launch_pdl(gelu_tanh_kernel<float>, blocks, threads, 0, stream, (const float*)in, (float*)out, (size_t)total);
  else if (dtype == RL_BF16)
    rl_launch_pdl(gelu_tanh_kernel<__nv_bfloat16>, blocks, threads, 0, stream, (const __nv_bfloat16*)in, (__nv_bfloat16*)out,
                  (size_t)total);
  else
    RL_REQUIRE(false, "rl_gelu_tanh: unknown dtype %d", dtype);
  RL_LAUNCH_CHECK("rl_gelu_tanh");
  return RL_OK;
}

// ------------------------------------------------------------------ additions to the residual between layers
// x[m, :] += (again ? again[m, :] : 0) + (vec ? vec[:] : 0), all float: what a model adds to the
// residual stream where a group of layers is entered (a copy of an earlier state of the stream,
// a learned vector of the pass).  The two are summed first, then added to x.
template <typename TV>
__global__ void residual_inject_kernel(float* __restrict__ x, const float* __restrict__ again,
                                       const TV* __restrict__ vec, size_t total, int d) {
  rl_pdl_trigger();
  rl_pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    float a = again ? again[i] : 0.f;
    if (vec) a += rl_ld(vec + (i % d));
    x[i] += a;
  }
}

extern "C" int rl_residual_inject(float* x, const float* again, const void* vec, int vec_dtype, int num_tokens,
                                  int hidden, cudaStream_t stream) {
  RL_REQUIRE(num_tokens >= 0 && hidden > 0, "rl_residual_inject: bad sizes M=%d d=%d", num_tokens, hidden);
  if (num_tokens == 0 || (again == nullptr && vec == nullptr)) return RL_OK;
  const size_t total = (size_t)num_tokens * hidden;
  const int threads = 256;
  const size_t want = (total + threads - 1) / threads;
  const int blocks = (int)(want < (size_t)rl_num_sms() * 16 ? want : (size_t)rl_num_sms() * 16);
  if (vec_dtype == RL_F32)
    rl_launch_pdl(residual_inject_kernel<float>, blocks, threads, 0, stream, x, again, (const float*)vec, total, hidden);
  else if (vec_dtype == RL_BF16)
    rl_launch_pdl(residual_inject_kernel<__nv_bfloat16>, blocks, threads, 0, stream, x, again, (const __nv_bfloat16*)vec, total, hidden);
  else
    RL_REQUIRE(false, "rl_residual_inject: unknown dtype %d", vec_dtype);
  RL_LAUNCH_CHECK("rl_residual_inject");
  return RL_OK;
}

// ------------------------------------------------------------------ soft cap of logits
// y = cap * tanh(y / cap) in place, float.
__global__ void softcap_kernel(float* __restrict__ y, size_t total, float cap, float inv_cap) {
  rl_pdl_trigger();
  rl_pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x)
    y[i] = cap * tanhf(y[i] * inv_cap);
}

extern "C" int rl_softcap(float* y, long long n, float cap, cudaStream_t stream) {
  RL_REQUIRE(n >= 0 && cap > 0.f, "rl_softcap: bad arguments n=%lld cap=%g", n, (double)cap);
  if (n == 0) return RL_OK;
  const int threads = 256;
  const long long want = (n + threads - 1) / threads;
  const int blocks = (int)(want < rl_num_sms() * 16 ? want : rl_num_sms() * 16);
  rl_launch_pdl(softcap_kernel, blocks, threads, 0, stream, y, (size_t)n, cap, 1.0f / cap);
  RL_LAUNCH_CHECK("rl_softcap");
  return RL_OK;
}

// ------------------------------------------------------------------ sigmoid gate
// y[m, i] *= 1 / (1 + exp(-g[m, i])) for i < n; the sigmoid in 32-bit.  g may be a view into a
// wider buffer (row stride ldg).
template <typename T>
__global__ void sigmoid_gate_kernel(T* __restrict__ y, int ldy, const T* __restrict__ g, int ldg, int M, int n) {
  rl_pdl_trigger();
  rl_pdl_wait();
  const size_t total = (size_t)M * n;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
    const size_t m = idx / n, i = idx % n;
    const float gate = 1.0f / (1.0f + expf(-rl_ld(g + m * ldg + i)));
    T* p = y + m * ldy + i;
    rl_st(p, rl_ld(p) * gate);
  }
}

// rows that 16-byte accesses can fetch (bf16): a block a row, eight elements a thread at a time
__global__ void __launch_bounds__(256)
sigmoid_gate_rows_kernel(__nv_bfloat16* __restrict__ y, int ldy, const __nv_bfloat16* __restrict__ g, int ldg, int n) {
  rl_pdl_trigger();
  rl_pdl_wait();
  __nv_bfloat16* yr = y + (size_t)blockIdx.x * ldy;
  const __nv_bfloat16* gr = g + (size_t)blockIdx.x * ldg;
  for (int i = 8 * threadIdx.x; i < n; i += 8 * 256) {
    uint4 yv = *reinterpret_cast<const uint4*>(yr + i);
    const uint4 gv = *reinterpret_cast<const uint4*>(gr + i);
    __nv_bfloat162* yp = reinterpret_cast<__nv_bfloat162*>(&yv);
    const __nv_bfloat162* gp = reinterpret_cast<const __nv_bfloat162*>(&gv);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 a = __bfloat1622float2(yp[k]), b = __bfloat1622float2(gp[k]);
      yp[k] = __floats2bfloat162_rn(a.x * (1.0f / (1.0f + expf(-b.x))), a.y * (1.0f / (1.0f + expf(-b.y))));
    }
    *reinterpret_cast<uint4*>(yr + i) = yv;
  }
}

extern "C" int rl_sigmoid_gate(void* y, int ldy, const void* g, int ldg, int dtype, int num_tokens, int n, cudaStream_t stream) {
  RL_REQUIRE(num_tokens >= 0 && n > 0 && ldy >= n && ldg >= n, "rl_sigmoid_gate: bad sizes M=%d n=%d", num_tokens, n);
  if (num_tokens == 0) return RL_OK;
  const size_t total = (size_t)num_tokens * n;
  const int threads = 256;
  const size_t want = (total + threads - 1) / threads;
  const int blocks = (int)(want < (size_t)rl_num_sms() * 16 ? want : (size_t)rl_num_sms() * 16);
  if (dtype == RL_BF16 && n % 8 == 0 && ldy % 8 == 0 && ldg % 8 == 0 && (((uintptr_t)y | (uintptr_t)g) & 15) == 0)
    rl_launch_pdl(sigmoid_gate_rows_kernel, num_tokens, 256, 0, stream, (__nv_bfloat16*)y, ldy, (const __nv_bfloat16*)g, ldg, n);
  else if (dtype == RL_F32)
    rl_launch_pdl(sigmoid_gate_kernel<float>, blocks, threads, 0, stream, (float*)y, ldy, (const float*)g, ldg, num_tokens, n);
  else if (dtype == RL_BF16)
    rl_launch_pdl(sigmoid_gate_kernel<__nv_bfloat16>, blocks, threads, 0, stream, (__nv_bfloat16*)y, ldy, (const __nv_bfloat16*)g, ldg, num_tokens, n);
  else
    RL_REQUIRE(false, "rl_sigmoid_gate: unknown dtype %d", dtype);
  RL_LAUNCH_CHECK("rl_sigmoid_gate");
  return RL_OK;
}

// ------------------------------------------------------------------ gated feed-forward with the tanh form of gelu
// out = gelu_tanh(gate) * up, for products that did not carry the activation in their epilogue (the 32-bit path,
// shapes the tensor-core product cannot address).  Layouts as for rl_swiglu.
template <typename T>
__global__ void geglu_kernel(const T* __restrict__ gu, T* __restrict__ out, int M, int I, int interleaved) {
  rl_pdl_trigger();
  rl_pdl_wait();
  const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (size_t)M * I) return;
  const size_t m = idx / I, i = idx % I;
  const T* row = gu + m * 2 * (size_t)I;
  const float g = rl_ld(interleaved ? row + 2 * i : row + i);
  const float u = rl_ld(interleaved ? row + 2 * i + 1 : row + I + i);
  const float act = 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
  rl_st(out + idx, act * u);
}

extern "C" int rl_geglu(const void* gate_up, void* out, int dtype, int num_tokens, int intermediate, int interleaved,
                        cudaStream_t stream) {
  RL_REQUIRE(num_tokens >= 0 && intermediate > 0, "rl_geglu: bad sizes M=%d I=%d", num_tokens, intermediate);
  if (num_tokens == 0) return RL_OK;
  const size_t total = (size_t)num_tokens * intermediate;
  const unsigned blocks = (unsigned)((total + 255) / 256);
  if (dtype == RL_F32)
    rl_launch_pdl(geglu_kernel<float>, blocks, 256, 0, stream, (const float*)gate_up, (float*)out, num_tokens, intermediate, interleaved);
  else if (dtype == RL_BF16)
    rl_launch_pdl(geglu_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, num_tokens,
                  intermediate, interleaved);
  else
    RL_REQUIRE(false, "rl_geglu: unknown dtype %d", dtype);
  RL_LAUNCH_CHECK("rl_geglu");
  return RL_OK;
}
