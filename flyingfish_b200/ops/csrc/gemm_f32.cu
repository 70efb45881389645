// FP32 linear layers on the CUDA cores, true 32-bit products:  Y[M,N] = act(X[M,K] · W[N,K]ᵀ + bias)
// For models run in 32-bit (comparisons, tests of a BF16 path); the BF16 linears are gemm_bf16.cu / gemm_skinny.cu.
// 64 x 64 tiles, 256 threads with 4 x 4 outputs each, K in steps of 16 through shared memory. The order of an output's
// additions is ascending k whatever M is.
#include "ptx.cuh"
#include "host_util.h"

namespace ff {

constexpr int F32_T = 64, F32_K = 16;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ X, const float* __restrict__ W, float* __restrict__ Y, int M, int N, int K, int ldx, int ldw,
                int ldy, const float* __restrict__ bias, int act) {
  pdl_trigger();
  pdl_wait();
  __shared__ __align__(16) float sx[F32_K][F32_T + 4];
  __shared__ __align__(16) float sw[F32_K][F32_T + 4];
  const int m0 = blockIdx.y * F32_T, n0 = blockIdx.x * F32_T;
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
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float v = acc[i][j] + (bias ? bias[n] : 0.f);
      if (act == 1) { v = fmaxf(v, 0.f); v *= v; }
      Y[(size_t)m * ldy + n] = v;
    }
  }
}

}  // namespace ff
using namespace ff;

FF_EXPORT int ff_gemm_f32(const float* X, const float* W, float* Y, int M, int N, int K, int ldx, int ldw, int ldy, const float* bias,
                          int act, cudaStream_t s) {
  if (M <= 0 || N <= 0 || K <= 0 || ldx < K || ldw < K || ldy < N || (unsigned)act > 1u) return FF_HOST_BAD_SHAPE;
  const long long my = (M + F32_T - 1) / F32_T;
  if (my > 65535) return FF_HOST_TOO_LARGE;
  if (int r = launch_pdl(gemm_f32_kernel, dim3((N + F32_T - 1) / F32_T, (unsigned)my), dim3(256), 0, s, 0, X, W, Y, M, N, K, ldx, ldw, ldy, bias, act)) return r;
  return launch_result();
}
