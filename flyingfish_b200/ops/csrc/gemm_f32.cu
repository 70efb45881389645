// FP32 linear layers on the CUDA cores, true 32-bit products:  Y[M,N] = act(X[M,K] · W[N,K]ᵀ + bias) * mul
// For models run in 32-bit (comparisons, tests of a BF16 path); the BF16 linears are gemm_bf16.cu / gemm_skinny.cu.
// 64 x 64 tiles, 256 threads with 4 x 4 outputs each, K in steps of 16 through shared memory. The order of an output's
// additions is ascending k whatever M is.
#include "ptx.cuh"
#include "host_util.h"

namespace ff {

constexpr int F32_T = 64, F32_K = 16;

// act 1: square of the positive part, 3: tanh-GELU; mul: a factor per element, row mul_rows[m] of a table of mul_table rows
struct F32Tail { const float* bias; int act; const float* mul; const int* mul_rows; int ldm, mul_table; };

// one 64 x 64 tile at (m0, n0)
__device__ __forceinline__ void gemm_f32_tile(const float* __restrict__ X, const float* __restrict__ W, float* __restrict__ Y, int m0, int n0,
                                              int M, int N, int K, int ldx, int ldw, int ldy, const F32Tail& tail) {
  __shared__ __align__(16) float sx[F32_K][F32_T + 4];
  __shared__ __align__(16) float sw[F32_K][F32_T + 4];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += F32_K) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + 256 * i, r = e >> 4, c = e & 15;
      sx[c][r] = (m0 + r < M && k0 + c < K) ? X[(size_t)(m0 + r) * ldx + k0 + c] : 0.f;
      sw[c][r] = (n0 + r < N && k0 + c < K) ? W[(size_t)(n0 + r) * ldw + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < F32_K; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sx[k][ty * 4]), b = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
    const float* f = nullptr;
    if (tail.mul != nullptr) {
      const int mr = tail.mul_rows[m];
      f = tail.mul + (size_t)(mr < 0 || mr >= tail.mul_table ? 0 : mr) * tail.ldm;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float v = acc[i][j] + (tail.bias ? tail.bias[n] : 0.f);
      if (tail.act == 1) { v = fmaxf(v, 0.f); v *= v; }
      if (tail.act == 3) v = 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
      if (f != nullptr) v *= f[n];
      Y[(size_t)m * ldy + n] = v;
    }
  }
}

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ X, const float* __restrict__ W, float* __restrict__ Y, int M, int N, int K, int ldx, int ldw,
                int ldy, const F32Tail tail, int a_cols, int c_cols) {
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.z;                                // block-diagonal product: head h (one head otherwise)
  gemm_f32_tile(X + (size_t)h * a_cols, W + (size_t)h * N * ldw, Y + (size_t)h * c_cols, blockIdx.y * F32_T, blockIdx.x * F32_T, M, N, K, ldx,
                ldw, ldy, tail);
}

// expert segments (seg_off / counts on the device): Y[segment rows, N] = X[segment rows, K] · W[e][N, K]ᵀ
__global__ void __launch_bounds__(256)
gemm_f32_grouped_kernel(const float* __restrict__ X, const float* __restrict__ W, float* __restrict__ Y, const int* __restrict__ seg_off,
                        const int* __restrict__ counts, int N, int K, int ldy, int capacity) {
  pdl_trigger();
  pdl_wait();
  const int e = blockIdx.y, r0 = seg_off[e];
  const int cnt = min(counts[e], capacity - r0);           // an overflowed dispatch is cut at the end of the buffers
  for (int m0 = blockIdx.z * F32_T; m0 < cnt; m0 += gridDim.z * F32_T)
    gemm_f32_tile(X + (size_t)r0 * K, W + (size_t)e * N * K, Y + (size_t)r0 * ldy, m0, blockIdx.x * F32_T, cnt, N, K, K, K, ldy, F32Tail{});
}

}  // namespace ff
using namespace ff;

FF_EXPORT int ff_gemm_f32(const float* X, const float* W, float* Y, int M, int N, int K, int ldx, int ldw, int ldy, const float* bias,
                          int act, const float* mul, const int* mul_rows, int ldm, int mul_table, cudaStream_t s) {
  if (M <= 0 || N <= 0 || K <= 0 || ldx < K || ldw < K || ldy < N || (act != 0 && act != 1 && act != 3)) return FF_HOST_BAD_SHAPE;
  if (mul != nullptr && (mul_rows == nullptr || mul_table < 1 || ldm < N)) return FF_HOST_BAD_SHAPE;
  const long long my = (M + F32_T - 1) / F32_T;
  if (my > 65535) return FF_HOST_TOO_LARGE;
  if (int r = launch_pdl(gemm_f32_kernel, dim3((N + F32_T - 1) / F32_T, (unsigned)my), dim3(256), 0, s, 0, X, W, Y, M, N, K, ldx, ldw, ldy,
                         F32Tail{bias, act, mul, mul_rows, ldm, mul_table}, 0, 0)) return r;
  return launch_result();
}

// Block-diagonal product: for every head h, Y[:, h * c_cols + (0..N)] = X[:, h * a_cols + (0..K)] · W[h]ᵀ with W [heads * N, K]
FF_EXPORT int ff_gemm_f32_heads(const float* X, const float* W, float* Y, int M, int heads, int N, int K, int ldx, int ldy, int a_cols, int c_cols,
                                cudaStream_t s) {
  if (M <= 0 || heads <= 0 || heads > 65535 || N <= 0 || K <= 0 || a_cols < K || c_cols < N) return FF_HOST_BAD_SHAPE;
  if (ldx < (heads - 1) * a_cols + K || ldy < (heads - 1) * c_cols + N) return FF_HOST_BAD_SHAPE;
  const long long my = (M + F32_T - 1) / F32_T;
  if (my > 65535) return FF_HOST_TOO_LARGE;
  if (int r = launch_pdl(gemm_f32_kernel, dim3((N + F32_T - 1) / F32_T, (unsigned)my, heads), dim3(256), 0, s, 0, X, W, Y, M, N, K, ldx, K, ldy,
                         F32Tail{}, a_cols, c_cols)) return r;
  return launch_result();
}

// Xs [capacity, K] contiguous rows, W [E * N, K], Y rows of ldy; segments as in ff_moe_grouped_gemm
FF_EXPORT int ff_gemm_f32_grouped(const float* Xs, const float* W, float* Y, const int* seg_off, const int* counts, int E, int N, int K,
                                  int capacity, int ldy, cudaStream_t s) {
  if (E <= 0 || E > 65535 || N <= 0 || K <= 0 || capacity <= 0 || ldy < N) return FF_HOST_BAD_SHAPE;
  int z = (capacity / E + F32_T - 1) / F32_T;
  if (z < 1) z = 1;
  if (z > 64) z = 64;
  if (int r = launch_pdl(gemm_f32_grouped_kernel, dim3((N + F32_T - 1) / F32_T, E, z), dim3(256), 0, s, 0, Xs, W, Y, seg_off, counts, N, K, ldy, capacity)) return r;
  return launch_result();
}
