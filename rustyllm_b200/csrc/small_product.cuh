// A small product for few tokens as a building block of kernels that do something with the sums at once:
// z[row, token] = sum_k w[row, k] * x[token, k] for SP_ROWS weight rows and up to 16 TW tokens, bf16 operands, float
// sums, on mma.sync m16n8k16.  A block of four warps: TW of them take 16 tokens each, the other factor 4 / TW cuts K
// (with few tokens the warps would otherwise idle); the parts of K are added in their order.  Both operands lie in shared
// memory whole (all loads in flight at once: a product of this size is one latency), rows padded by 8 elements so that
// ldmatrix meets no bank twice, columns beyond K zero up to a multiple of 16.
#pragma once
#include "common.cuh"

#define SP_ROWS 32
#define SP_THREADS 128

__device__ __forceinline__ void sp_cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void sp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void sp_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
__device__ __forceinline__ void sp_ldm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sp_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Shared memory: weights [SP_ROWS][ld] bf16, tokens [16 TW][ld] bf16, sums [4 / TW][SP_ROWS][16 TW + 1] float.
struct SpLayout {
  int kp, ld;                        // K rounded up to 16; elements from row to row
  uint32_t x_off, z_off, bytes;
};
__host__ __device__ inline SpLayout sp_layout(int K, int TW) {
  SpLayout L;
  L.kp = (K + 15) & ~15;
  L.ld = L.kp + 8;
  L.x_off = SP_ROWS * L.ld * 2;
  L.z_off = L.x_off + 16 * TW * L.ld * 2;
  L.bytes = L.z_off + (4 / TW) * SP_ROWS * (16 * TW + 1) * 4;
  return L;
}
static inline int sp_token_warps(int M) { return M <= 16 ? 1 : M <= 32 ? 2 : 4; }

// Requests rows of K bf16 elements (a multiple of 8, every row 16-byte aligned); row r < have comes from row_ptr(r), the
// others and the columns beyond K are zero.  The caller commits and waits.
template <typename RowPtr>
__device__ __forceinline__ void sp_fetch(uint8_t* smem, uint32_t off, int rows, int have, int K, const SpLayout& L, RowPtr row_ptr) {
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem) + off;
  const int pieces = L.kp >> 3;
  for (int i = threadIdx.x; i < rows * pieces; i += SP_THREADS) {
    const int r = i / pieces, ch = i - r * pieces;
    if (r < have && ch * 8 < K) sp_cp16(base + (uint32_t)(r * L.ld * 2 + ch * 16), row_ptr(r) + ch * 8);
    else *reinterpret_cast<uint4*>(smem + off + r * L.ld * 2 + ch * 16) = make_uint4(0u, 0u, 0u, 0u);
  }
}

// After the fetches have landed for all threads: the sums of this block; complete for everyone on return.
// sp_sum reads one.
template <int TW>
__device__ __forceinline__ void sp_multiply(uint8_t* smem, const SpLayout& L) {
  constexpr int KW = 4 / TW, ZT = 16 * TW + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int tw = warp % TW, kw = warp / TW;
  const int r8 = lane & 7, mat = lane >> 3;
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem);
  const uint32_t wa = base + (uint32_t)(((r8 + 8 * (mat & 1)) * L.ld + 8 * (mat >> 1)) * 2);
  const uint32_t xa = base + L.x_off + (uint32_t)(((16 * tw + r8 + 8 * (mat >> 1)) * L.ld + 8 * (mat & 1)) * 2);
  float acc[2][2][4];
#pragma unroll
  for (int a = 0; a < 2; ++a)
#pragma unroll
    for (int b = 0; b < 2; ++b) acc[a][b][0] = acc[a][b][1] = acc[a][b][2] = acc[a][b][3] = 0.f;
  for (int k = 16 * kw; k < L.kp; k += 16 * KW) {
    uint32_t w0[4], w1[4], x[4];
    sp_ldm4(w0, wa + k * 2);
    sp_ldm4(w1, wa + (uint32_t)(16 * L.ld * 2) + k * 2);
    sp_ldm4(x, xa + k * 2);
    sp_mma(acc[0][0], w0, x[0], x[1]);
    sp_mma(acc[0][1], w0, x[2], x[3]);
    sp_mma(acc[1][0], w1, x[0], x[1]);
    sp_mma(acc[1][1], w1, x[2], x[3]);
  }
  float* z = reinterpret_cast<float*>(smem + L.z_off) + kw * SP_ROWS * ZT;
#pragma unroll
  for (int a = 0; a < 2; ++a)
#pragma unroll
    for (int b = 0; b < 2; ++b)
#pragma unroll
      for (int e = 0; e < 4; ++e) z[(16 * a + g + 8 * (e >> 1)) * ZT + 16 * tw + 8 * b + 2 * t + (e & 1)] = acc[a][b][e];
  __syncthreads();
}
template <int TW>
__device__ __forceinline__ float sp_sum(const uint8_t* smem, const SpLayout& L, int row, int token) {
  constexpr int KW = 4 / TW, ZT = 16 * TW + 1;
  const float* z = reinterpret_cast<const float*>(smem + L.z_off) + row * ZT + token;
  float v = z[0];
#pragma unroll
  for (int k = 1; k < KW; ++k) v += z[k * SP_ROWS * ZT];
  return v;
}
