// Residual streams with fixed hyper-connections. A row holds `S` FP32 streams x_0..x_{S-1} of `width` elements.
//   embed : x_s = table[id] * scale for every s;   n = rmsnorm(sum_s a_s x_s) * w
//   step  : x_t <- sum_s M[s, t] x_s + b_t (y * c);   n = rmsnorm(sum_t a_t x_t) * w
// The step is the write of one sub-layer (y its result, c a factor per channel, b and M its coefficients), the read of
// the next one (a) and that one's norm: every stream element is read once and written once, the sub-layer's input
// leaves as the GEMM operand. One block per row; a thread owns the same columns of all streams, so the update is in
// place. The last sub-layer of a model does not write the streams back. Memory bound: (2 S + 1) FP32-equivalents plus
// y and n per element.
// mhc.cu has the form whose coefficients are computed from the streams.
#include "dtype_io.cuh"
#include "host_util.h"

namespace ff {

constexpr int ST_MAX = 16;
constexpr int ST_THREADS = 512;

// MS: streams held per thread; EXACT: MS is the number of streams, otherwise `streams` <= MS is
template <typename T, int MS, bool EXACT, bool EMBED>
__global__ void __launch_bounds__(ST_THREADS)
stream_kernel(const int* __restrict__ ids, const T* __restrict__ table, float scale, int vocab, float* __restrict__ x,
              const T* __restrict__ y, const T* __restrict__ chan, const float* __restrict__ coef, const T* __restrict__ norm_w,
              T* __restrict__ n, int streams, int width, int true_width, float eps, int write, int* status) {
  pdl_trigger();
  extern __shared__ __align__(16) float st_u[];            // [width] the next sub-layer's input before its norm
  __shared__ float s_coef[ST_MAX * (ST_MAX + 2)];
  __shared__ float s_red[ST_THREADS / 32];
  const int S = EXACT ? MS : streams;
  const int row = blockIdx.x, tid = threadIdx.x;
  const int ncoef = EMBED ? S : S * (S + 2);
  for (int i = tid; i < ncoef; i += blockDim.x) s_coef[i] = coef[i];      // weights: written by no kernel
  __syncthreads();
  pdl_wait();
  const T* src = nullptr;
  if (EMBED) {
    int id = ids[row];
    if (id < 0 || id >= vocab) { if (tid == 0) set_status(status, KID_EMBED, FF_ERR_BOUNDS, row, id); id = 0; }
    src = table + (size_t)id * width;
  } else {
    src = y + (size_t)row * width;
  }
  float* xr = x + (size_t)row * S * width;
  const float* ca = s_coef, * cb = s_coef + S, * cm = s_coef + 2 * S;
  float ss = 0.f;
  for (int c = tid * 4; c < width; c += blockDim.x * 4) {
    float in[4], u[4] = {0.f, 0.f, 0.f, 0.f};
    load4(src + c, in);
    if (EMBED) {
      float asum = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) in[j] *= scale;
#pragma unroll
      for (int s = 0; s < MS; ++s)
        if (EXACT || s < S) { store4(xr + (size_t)s * width + c, in); asum += ca[s]; }
#pragma unroll
      for (int j = 0; j < 4; ++j) u[j] = asum * in[j];
    } else {
      float k[4], old[MS][4];
#pragma unroll
      for (int s = 0; s < MS; ++s)
        if (EXACT || s < S) load4(xr + (size_t)s * width + c, old[s]);
      load4(chan + c, k);
#pragma unroll
      for (int j = 0; j < 4; ++j) in[j] *= k[j];
#pragma unroll
      for (int t = 0; t < MS; ++t)
        if (EXACT || t < S) {
          float v[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) v[j] = cb[t] * in[j];
#pragma unroll
          for (int s = 0; s < MS; ++s)
            if (EXACT || s < S) {
              const float m = cm[s * S + t];
#pragma unroll
              for (int j = 0; j < 4; ++j) v[j] = fmaf(m, old[s][j], v[j]);
            }
          if (write) store4(xr + (size_t)t * width + c, v);
#pragma unroll
          for (int j = 0; j < 4; ++j) u[j] = fmaf(ca[t], v[j], u[j]);
        }
    }
    store4(st_u + c, u);
#pragma unroll
    for (int j = 0; j < 4; ++j) ss = fmaf(u[j], u[j], ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) s_red[tid >> 5] = ss;
  __syncthreads();
  float tot = (tid & 31) < (int)(blockDim.x >> 5) ? s_red[tid & 31] : 0.f;
  tot = warp_sum(tot);
  const float r = 1.0f / sqrtf(tot / (float)true_width + eps);
  for (int c = tid * 4; c < width; c += blockDim.x * 4) {      // the thread's own columns again
    float u[4], w[4];
    load4(st_u + c, u);
    load4(norm_w + c, w);
#pragma unroll
    for (int j = 0; j < 4; ++j) u[j] = u[j] * r * w[j];
    store4(n + (size_t)row * width + c, u);
  }
}

template <typename T, bool EMBED>
static int stream_launch(const int* ids, const T* table, float scale, int vocab, float* x, const T* y, const T* chan, const float* coef,
                         const T* norm_w, T* n, int rows, int streams, int width, int true_width, float eps, int write, int* status,
                         cudaStream_t s) {
  if (rows <= 0 || streams < 1 || streams > ST_MAX || width <= 0 || width % 8 || true_width <= 0 || true_width > width) return FF_HOST_BAD_SHAPE;
  const int smem = width * 4;
  if (smem > 200 * 1024) return FF_HOST_TOO_LARGE;
  int threads = (width / 4 + 31) / 32 * 32;
  // a few rows (a decode step): wide blocks, for latency; many: more, smaller blocks per SM keep more loads in flight
  const int cap = rows >= 2 * sm_count() ? ST_THREADS / 2 : ST_THREADS;
  if (threads > cap) threads = cap;
  auto go = [&](auto kern) -> int {
    if (int r = opt_in_smem(kern, smem)) return r;
    if (int r = launch_pdl(kern, dim3(rows), dim3(threads), smem, s, 0, ids, table, scale, vocab, x, y, chan, coef, norm_w, n, streams,
                           width, true_width, eps, write, status)) return r;
    return launch_result();
  };
  switch (streams) {
    case 1: return go(stream_kernel<T, 1, true, EMBED>);
    case 2: return go(stream_kernel<T, 2, true, EMBED>);
    case 3: return go(stream_kernel<T, 3, true, EMBED>);
    case 4: return go(stream_kernel<T, 4, true, EMBED>);
    default: break;
  }
  if (streams <= 8) return go(stream_kernel<T, 8, false, EMBED>);
  return go(stream_kernel<T, 16, false, EMBED>);
}

}  // namespace ff
using namespace ff;

// table [vocab, width] and norm_w, n in BF16 (f32 = 0) or FP32; read float[S]; x FP32 [rows, S, width]
FF_EXPORT int ff_stream_embed(const int* ids, const void* table, float scale, const float* read, const void* norm_w, float* x, void* n,
                              int rows, int streams, int width, int true_width, int vocab, float eps, int f32, int* status, cudaStream_t s) {
  if (f32)
    return stream_launch<float, true>(ids, (const float*)table, scale, vocab, x, nullptr, nullptr, read, (const float*)norm_w, (float*)n, rows,
                                      streams, width, true_width, eps, 1, status, s);
  return stream_launch<__nv_bfloat16, true>(ids, (const __nv_bfloat16*)table, scale, vocab, x, nullptr, nullptr, read,
                                            (const __nv_bfloat16*)norm_w, (__nv_bfloat16*)n, rows, streams, width, true_width, eps, 1, status, s);
}

// coef float[S * (S + 2)]: read of the next sub-layer, write, matrix [from, to]
FF_EXPORT int ff_stream_step(float* x, const void* y, const void* chan, const float* coef, const void* norm_w, void* n, int rows, int streams,
                             int width, int true_width, float eps, int f32, int write, cudaStream_t s) {
  if (f32)
    return stream_launch<float, false>(nullptr, nullptr, 1.f, 0, x, (const float*)y, (const float*)chan, coef, (const float*)norm_w, (float*)n,
                                       rows, streams, width, true_width, eps, write, nullptr, s);
  return stream_launch<__nv_bfloat16, false>(nullptr, nullptr, 1.f, 0, x, (const __nv_bfloat16*)y, (const __nv_bfloat16*)chan, coef,
                                             (const __nv_bfloat16*)norm_w, (__nv_bfloat16*)n, rows, streams, width, true_width, eps, write,
                                             nullptr, s);
}
