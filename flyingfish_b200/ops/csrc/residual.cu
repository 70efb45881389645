// FP32 residual stream of layers whose mixer and feed-forward read the same rows through two norms (parallel layers):
//   embed : x = table[id] * scale
//   step  : x += a + b + sum_j w_j y_j          a, b: rows of the mixer and of a dense or shared feed-forward
// With inner norms (a second mixer beside the first, embeddings of bigrams beside those of tokens):
//   embed : x = t / rms(t) * w,  t = table[id] + table2[id2]         bigram_rows: id2 from the token and the one before it
//   step  : x += a / rms(a) * wa + a2 / rms(a2) * wa2 + b + ..
//   n1 = x / rms(x) * w1     n2 = x / rms(x) * w2      the operands of the next layer (n2 optional)
// The sum over a row's chosen experts is taken here, straight from the rows the grouped GEMM wrote (y_j = y[pos_j]; a choice
// beyond the last expert is an identity output: y_j is the row h the experts were given), so a layer ends in one kernel: the
// residual is read and written once in FP32 and nothing is rounded on the way. One block per row; a thread owns the same
// columns in both passes. Norm weights are FP32 (offsets already added).
//
// Layers whose sub-layers are normed on both sides (sequential layers) have a kernel of their own below:
//   x += inner(y)        n = outer(x)
// inner is the norm behind a sub-layer, outer the one in front of the next: an RMS norm, or tanh(alpha x) w + b (which needs no
// statistics of the row); outer may also be a plain copy in the GEMM operand's type.
#include "dtype_io.cuh"
#include "host_util.h"
#include <type_traits>

namespace ff {

constexpr int RN_THREADS = 512;
constexpr int RN_TOP_MAX = 32;

// the chosen experts' contributions of a row; top == 0: none
template <typename T>
struct ExpertRows {
  const T* y; const int* pos; const int* ids; const float* w; const T* h;
  int top, experts, ldy;
};

// inner norms; t2, rows2: the second table and its row per row of the batch (embed), a2: rows of the second mixer (step)
template <typename T>
struct InnerNorms { const T* t2; const int* rows2; int rows_t2; const T* a2; const float* w; const float* w2; };

// all threads of the block: one over the root mean square from the threads' sums of squares
__device__ __forceinline__ float block_rms(float ss, float* s_red, int true_width, float eps) {
  ss = warp_sum(ss);
  __syncthreads();                                         // the previous reduction has been read
  if ((threadIdx.x & 31) == 0) s_red[threadIdx.x >> 5] = ss;
  __syncthreads();
  const float tot = warp_sum((threadIdx.x & 31) < (blockDim.x >> 5) ? s_red[threadIdx.x & 31] : 0.f);
  return 1.0f / sqrtf(tot / (float)true_width + eps);
}

template <typename T, bool EMBED, bool INNER>
__global__ void __launch_bounds__(RN_THREADS)
residual_norms_kernel(float* __restrict__ x, const int* __restrict__ ids, const T* __restrict__ table, float scale, int vocab,
                      const T* __restrict__ a, const T* __restrict__ b, const ExpertRows<T> ex, const InnerNorms<T> in, const float* __restrict__ w1,
                      const float* __restrict__ w2, T* __restrict__ n1, T* __restrict__ n2, int width, int true_width, float eps,
                      int* status) {
  pdl_trigger();
  extern __shared__ __align__(16) float rn_x[];            // [width] the row between the two passes
  __shared__ const T* s_src[RN_TOP_MAX];
  __shared__ float s_w[RN_TOP_MAX];
  __shared__ float s_red[RN_THREADS / 32];
  const int row = blockIdx.x, tid = threadIdx.x;
  pdl_wait();
  const T* src = nullptr;
  if (EMBED) {
    int id = ids[row];
    if (id < 0 || id >= vocab) { if (tid == 0) set_status(status, KID_EMBED, FF_ERR_BOUNDS, row, id); id = 0; }
    src = table + (size_t)id * width;
  } else if (ex.top > 0) {
    if (tid < ex.top) {
      const int i = row * ex.top + tid, e = ex.ids[i], p = ex.pos[i];
      s_src[tid] = e >= ex.experts ? ex.h + (size_t)row * width : (p >= 0 ? ex.y + (size_t)p * ex.ldy : nullptr);
      s_w[tid] = ex.w[i];
    }
    __syncthreads();
  }
  float* xr = x + (size_t)row * width;
  float ra = 1.f, ra2 = 1.f;
  const T* src2 = nullptr;
  if constexpr (INNER) {
    const T* one = EMBED ? src : a + (size_t)row * width;
    if (EMBED) {
      int r2 = in.rows2[row];
      if (r2 < 0 || r2 >= in.rows_t2) { if (tid == 0) set_status(status, KID_EMBED, FF_ERR_BOUNDS, row, r2); r2 = 0; }
      src2 = in.t2 + (size_t)r2 * width;
    } else {
      src2 = in.a2 + (size_t)row * width;
    }
    float s1 = 0.f, s2 = 0.f;
    for (int c = tid * 4; c < width; c += blockDim.x * 4) {
      float u[4], t[4];
      load4(one + c, u);
      load4(src2 + c, t);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (EMBED) u[j] = u[j] * scale + t[j];
        s1 = fmaf(u[j], u[j], s1);
        s2 = fmaf(t[j], t[j], s2);
      }
    }
    ra = block_rms(s1, s_red, true_width, eps);
    if (!EMBED) ra2 = block_rms(s2, s_red, true_width, eps);
    __syncthreads();
  }
  float ss = 0.f;
  for (int c = tid * 4; c < width; c += blockDim.x * 4) {
    float v[4];
    if (EMBED) {
      load4(src + c, v);
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] *= scale;
      if constexpr (INNER) {
        float t[4], f[4];
        load4(src2 + c, t);
        load4(in.w + c, f);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] = (v[j] + t[j]) * ra * f[j];
      }
    } else {
      float t[4];
      load4(xr + c, v);
      load4(a + (size_t)row * width + c, t);
      if constexpr (INNER) {
        float f[4], u[4], f2[4];
        load4(in.w + c, f);
        load4(src2 + c, u);
        load4(in.w2 + c, f2);
#pragma unroll
        for (int j = 0; j < 4; ++j) t[j] = t[j] * ra * f[j] + u[j] * ra2 * f2[j];
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] += t[j];
      if (b != nullptr) {
        load4(b + (size_t)row * width + c, t);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] += t[j];
      }
      for (int k = 0; k < ex.top; ++k) {
        const T* p = s_src[k];
        if (p == nullptr) continue;                        // not served (overflow, reported by the dispatch)
        load4(p + c, t);
        const float w = s_w[k];
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] = fmaf(w, t[j], v[j]);
      }
    }
    store4(xr + c, v);
    store4(rn_x + c, v);
#pragma unroll
    for (int j = 0; j < 4; ++j) ss = fmaf(v[j], v[j], ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) s_red[tid >> 5] = ss;
  __syncthreads();
  float tot = (tid & 31) < (int)(blockDim.x >> 5) ? s_red[tid & 31] : 0.f;
  tot = warp_sum(tot);
  const float r = 1.0f / sqrtf(tot / (float)true_width + eps);
  for (int c = tid * 4; c < width; c += blockDim.x * 4) {      // the thread's own columns again
    float v[4], w[4], o[4];
    load4(rn_x + c, v);
    load4(w1 + c, w);
#pragma unroll
    for (int j = 0; j < 4; ++j) { v[j] *= r; o[j] = v[j] * w[j]; }
    store4(n1 + (size_t)row * width + c, o);
    if (w2 != nullptr) {
      load4(w2 + c, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = v[j] * w[j];
      store4(n2 + (size_t)row * width + c, o);
    }
  }
}

// rows of a second embedding table: (previous token * mul_prev + token * mul_cur) mod buckets, `buckets` for a sequence's first token.
// The previous token of a sequence's first new row is its state (negative: none), which then takes the last one. A block per sequence.
__global__ void __launch_bounds__(256)
bigram_rows_kernel(const int* __restrict__ ids, int* __restrict__ out, int* __restrict__ last, const int* __restrict__ row_start,
                   const int* __restrict__ slots, int buckets, long long mul_prev, long long mul_cur) {
  pdl_trigger();
  pdl_wait();
  const int r0 = row_start[blockIdx.x], r1 = row_start[blockIdx.x + 1], slot = slots[blockIdx.x];
  if (r1 <= r0) return;
  for (int r = r0 + threadIdx.x; r < r1; r += blockDim.x) {
    const int before = r == r0 ? last[slot] : max(ids[r - 1], 0);     // ids outside the vocabulary are reported by the embedding
    out[r] = before < 0 ? buckets : (int)((before * mul_prev + max(ids[r], 0) * mul_cur) % buckets);
  }
  if (threadIdx.x == 0) last[slot] = ids[r1 - 1];          // the thread that read it
}

template <typename T, bool EMBED, bool INNER>
static int residual_launch(float* x, const int* ids, const void* table, float scale, int vocab, const void* a, const void* b,
                           const ExpertRows<T>& ex, const InnerNorms<T>& in, const float* w1, const float* w2, void* n1, void* n2, int rows, int width, int true_width,
                           float eps, int* status, cudaStream_t s) {
  if (rows <= 0 || width <= 0 || width % 8 || true_width <= 0 || true_width > width || (w2 == nullptr) != (n2 == nullptr)) return FF_HOST_BAD_SHAPE;
  if (ex.top < 0 || ex.top > RN_TOP_MAX || (ex.top > 0 && (ex.ldy % 8 || ex.pos == nullptr || ex.ids == nullptr || ex.w == nullptr))) return FF_HOST_BAD_SHAPE;
  const int smem = width * 4;
  if (smem > 200 * 1024) return FF_HOST_TOO_LARGE;
  if ((reinterpret_cast<uintptr_t>(in.w) & 15) || (reinterpret_cast<uintptr_t>(in.w2) & 15)) return FF_HOST_BAD_ALIGN;
  if (INNER && (in.w == nullptr || (EMBED ? in.t2 == nullptr || in.rows2 == nullptr : in.a2 == nullptr || in.w2 == nullptr))) return FF_HOST_BAD_SHAPE;
  auto kern = residual_norms_kernel<T, EMBED, INNER>;
  if (int r = opt_in_smem(kern, smem)) return r;
  int threads = (width / 4 + 31) / 32 * 32;
  // a few rows (a decode step): wide blocks, for latency; many: more, smaller blocks per SM keep more loads in flight
  const int cap = rows >= 2 * sm_count() ? RN_THREADS / 2 : RN_THREADS;
  if (threads > cap) threads = cap;
  if (int r = launch_pdl(kern, dim3(rows), dim3(threads), smem, s, 0, x, ids, (const T*)table, scale, vocab, (const T*)a, (const T*)b, ex, in, w1,
                         w2, (T*)n1, (T*)n2, width, true_width, eps, status)) return r;
  return launch_result();
}

// ------------------------------------------------------------------------------------------
// norms on both sides of a sub-layer
// ------------------------------------------------------------------------------------------
enum { NORM_COPY = 0, NORM_RMS = 1, NORM_TANH = 2 };

struct NormArgs { const float* w; const float* b; float alpha; int kind; };

// BF16 results: 1 - 2 / (1 + e^2x), whose error (1e-7 of 1) vanishes in the rounding; FP32 results take tanhf
__device__ __forceinline__ float norm_tanh(float x, __nv_bfloat16) { return 1.0f - __fdividef(2.0f, 1.0f + __expf(2.0f * fminf(x, 20.0f))); }
__device__ __forceinline__ float norm_tanh(float x, float) { return tanhf(x); }

// four columns at c: v <- norm(v); r: one over the row's root mean square (RMS norm)
template <typename T>
__device__ __forceinline__ void apply_norm(const NormArgs& a, int c, float r, float (&v)[4]) {
  if (a.kind == NORM_COPY) return;
  float w[4];
  load4(a.w + c, w);
  if (a.kind == NORM_RMS) {
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = v[j] * r * w[j];
    return;
  }
  float b[4];
  load4(a.b + c, b);
#pragma unroll
  for (int j = 0; j < 4; ++j) v[j] = fmaf(norm_tanh(a.alpha * v[j], T()), w[j], b[j]);
}

template <typename T, bool EMBED>
__global__ void __launch_bounds__(RN_THREADS)
residual_sandwich_kernel(float* __restrict__ x, const int* __restrict__ ids, const T* __restrict__ table, float scale, int vocab,
                         const T* __restrict__ y, NormArgs inner, NormArgs outer, T* __restrict__ n, int width, int true_width, float eps,
                         int* status) {
  pdl_trigger();
  extern __shared__ __align__(16) float rn_x[];            // [width] the row between passes (only with an RMS norm)
  __shared__ float s_red[RN_THREADS / 32];
  const int row = blockIdx.x, tid = threadIdx.x, step = blockDim.x * 4;
  pdl_wait();
  const T* src;
  if (EMBED) {
    int id = ids[row];
    if (id < 0 || id >= vocab) { if (tid == 0) set_status(status, KID_EMBED, FF_ERR_BOUNDS, row, id); id = 0; }
    src = table + (size_t)id * width;
  } else {
    src = y + (size_t)row * width;
  }
  float* xr = x + (size_t)row * width;
  T* nr = n + (size_t)row * width;
  float r_in = 1.f;
  const bool stage = !EMBED && inner.kind == NORM_RMS;
  if (stage) {
    float ss = 0.f;
    for (int c = tid * 4; c < width; c += step) {
      float t[4];
      load4(src + c, t);
      store4(rn_x + c, t);
#pragma unroll
      for (int j = 0; j < 4; ++j) ss = fmaf(t[j], t[j], ss);
    }
    r_in = block_rms(ss, s_red, true_width, eps);
  }
  float ss = 0.f;
  for (int c = tid * 4; c < width; c += step) {
    float v[4];
    if (EMBED) {
      load4(src + c, v);
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] *= scale;
    } else {
      float t[4];
      load4(xr + c, v);
      if (stage) load4(rn_x + c, t); else load4(src + c, t);
      apply_norm<T>(inner, c, r_in, t);
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] += t[j];
    }
    store4(xr + c, v);
    if (outer.kind == NORM_RMS) {
      store4(rn_x + c, v);
#pragma unroll
      for (int j = 0; j < 4; ++j) ss = fmaf(v[j], v[j], ss);
    } else {
      apply_norm<T>(outer, c, 1.f, v);
      store4(nr + c, v);
    }
  }
  if (outer.kind != NORM_RMS) return;
  const float r = block_rms(ss, s_red, true_width, eps);
  for (int c = tid * 4; c < width; c += step) {            // the thread's own columns again
    float v[4];
    load4(rn_x + c, v);
    apply_norm<T>(outer, c, r, v);
    store4(nr + c, v);
  }
}

template <typename T, bool EMBED>
static int sandwich_launch(float* x, const int* ids, const void* table, float scale, int vocab, const void* y, NormArgs inner, NormArgs outer,
                           void* n, int rows, int width, int true_width, float eps, int* status, cudaStream_t s) {
  if (rows <= 0 || width <= 0 || width % 8 || true_width <= 0 || true_width > width) return FF_HOST_BAD_SHAPE;
  for (const NormArgs* a : {&inner, &outer}) {
    if ((unsigned)a->kind > NORM_TANH || (a->kind != NORM_COPY && a->w == nullptr) || (a->kind == NORM_TANH && a->b == nullptr)) return FF_HOST_BAD_SHAPE;
    if ((reinterpret_cast<uintptr_t>(a->w) & 15) || (reinterpret_cast<uintptr_t>(a->b) & 15)) return FF_HOST_BAD_ALIGN;
  }
  const int smem = inner.kind == NORM_RMS || outer.kind == NORM_RMS ? width * 4 : 0;
  if (smem > 200 * 1024) return FF_HOST_TOO_LARGE;
  auto kern = residual_sandwich_kernel<T, EMBED>;
  if (int r = opt_in_smem(kern, smem)) return r;
  int threads = (width / 4 + 31) / 32 * 32;
  const int cap = rows >= 2 * sm_count() ? RN_THREADS / 2 : RN_THREADS;
  if (threads > cap) threads = cap;
  if (int r = launch_pdl(kern, dim3(rows), dim3(threads), smem, s, 0, x, ids, (const T*)table, scale, vocab, (const T*)y, inner, outer, (T*)n,
                         width, true_width, eps, status)) return r;
  return launch_result();
}

}  // namespace ff
using namespace ff;

// x FP32 [rows, width] = table[id] * scale; n = outer(x). kinds: 0 copy, 1 RMS norm times w, 2 tanh(alpha x) w + b; w, b FP32 [width]
FF_EXPORT int ff_residual_embed_normed(const int* ids, const void* table, float scale, float* x, int kind, const float* w, const float* b,
                                       float alpha, void* n, int rows, int width, int true_width, int vocab, float eps, int f32, int* status,
                                       cudaStream_t s) {
  const NormArgs none = {nullptr, nullptr, 0.f, NORM_COPY}, outer = {w, b, alpha, kind};
  if (f32) return sandwich_launch<float, true>(x, ids, table, scale, vocab, nullptr, none, outer, n, rows, width, true_width, eps, status, s);
  return sandwich_launch<__nv_bfloat16, true>(x, ids, table, scale, vocab, nullptr, none, outer, n, rows, width, true_width, eps, status, s);
}

// x += inner(y); n = outer(x)
FF_EXPORT int ff_residual_add_normed(float* x, const void* y, int ikind, const float* iw, const float* ib, float ialpha, int okind, const float* ow,
                                     const float* ob, float oalpha, void* n, int rows, int width, int true_width, float eps, int f32,
                                     cudaStream_t s) {
  const NormArgs inner = {iw, ib, ialpha, ikind}, outer = {ow, ob, oalpha, okind};
  if (f32) return sandwich_launch<float, false>(x, nullptr, nullptr, 1.f, 0, y, inner, outer, n, rows, width, true_width, eps, nullptr, s);
  return sandwich_launch<__nv_bfloat16, false>(x, nullptr, nullptr, 1.f, 0, y, inner, outer, n, rows, width, true_width, eps, nullptr, s);
}

// x FP32 [rows, width]; table, n1, n2 in BF16 (f32 = 0) or FP32; w1, w2 FP32 [width] (w2, n2: both or neither). table2 [rows_t2, width],
// rows2 [rows], w_in FP32 [width]: the second table and the norm of the sum, or null
FF_EXPORT int ff_residual_embed(const int* ids, const void* table, float scale, const void* table2, const int* rows2, int rows_t2, const float* w_in,
                                float* x, const float* w1, const float* w2, void* n1, void* n2, int rows, int width, int true_width, int vocab,
                                float eps, int f32, int* status, cudaStream_t s) {
  auto go = [&](auto* t) -> int {
    using T = std::remove_pointer_t<decltype(t)>;
    const InnerNorms<T> in = {(const T*)table2, rows2, rows_t2, nullptr, w_in, nullptr};
    if (table2 != nullptr)
      return residual_launch<T, true, true>(x, ids, table, scale, vocab, nullptr, nullptr, ExpertRows<T>{}, in, w1, w2, n1, n2, rows, width, true_width, eps, status, s);
    return residual_launch<T, true, false>(x, ids, table, scale, vocab, nullptr, nullptr, ExpertRows<T>{}, in, w1, w2, n1, n2, rows, width, true_width, eps, status, s);
  };
  return f32 ? go((float*)nullptr) : go((__nv_bfloat16*)nullptr);
}

// a: [rows, width]; a2: the same or null, then wa and wa2 FP32 [width] are the weights of the norms of both; b: the same or null; y, pos,
// eids, ew, h: the experts' rows, the row of every choice (negative: none), the choices [rows, top] and weights, and the experts' input
// (top = 0: no experts)
FF_EXPORT int ff_residual_step(float* x, const void* a, const void* a2, const float* wa, const float* wa2, const void* b, const void* y,
                               const int* pos, const int* eids, const float* ew, const void* h, int top, int experts, int ldy, const float* w1,
                               const float* w2, void* n1, void* n2, int rows, int width, int true_width, float eps, int f32, cudaStream_t s) {
  auto go = [&](auto* t) -> int {
    using T = std::remove_pointer_t<decltype(t)>;
    const ExpertRows<T> ex = {(const T*)y, pos, eids, ew, (const T*)h, top, experts, ldy};
    const InnerNorms<T> in = {nullptr, nullptr, 0, (const T*)a2, wa, wa2};
    if (a2 != nullptr)
      return residual_launch<T, false, true>(x, nullptr, nullptr, 1.f, 0, a, b, ex, in, w1, w2, n1, n2, rows, width, true_width, eps, nullptr, s);
    return residual_launch<T, false, false>(x, nullptr, nullptr, 1.f, 0, a, b, ex, in, w1, w2, n1, n2, rows, width, true_width, eps, nullptr, s);
  };
  return f32 ? go((float*)nullptr) : go((__nv_bfloat16*)nullptr);
}

// ids int[rows], out int[rows], last int[slots]
FF_EXPORT int ff_bigram_rows(const int* ids, int* out, int* last, const int* row_start, const int* slots, int sequences, int buckets,
                             long long mul_prev, long long mul_cur, cudaStream_t s) {
  if (sequences <= 0 || buckets < 1 || mul_prev < 0 || mul_cur < 0) return FF_HOST_BAD_SHAPE;
  if (int r = launch_pdl(bigram_rows_kernel, dim3(sequences), dim3(256), 0, s, 0, ids, out, last, row_start, slots, buckets, mul_prev, mul_cur)) return r;
  return launch_result();
}
