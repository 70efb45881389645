// Per-head RMS norm of packed projection rows, rotation of neighbouring elements, value blending, and the paged-cache write
// (rotate-half positions without a norm: rope_kv_paged in rope_act_sample.cu).
//   row = [hq query heads | hkv key heads | hkv value heads | ...], heads `dk` / `dv` elements apart of which the first
//   `dim` count for the norm (the rest is zero padding)
//   q <- rot(q / rms(q) * wq)            in the row         (weights and rotation where they are given: neighbours 2i, 2i + 1 of
//   k <- rot(k / rms(k) * wk)            to its slot         the first elements turn by the row's table of cosines and sines)
//                                        to its slot of the K cache [block][kv head][block_size][dk]
//   v <- (1 - mix) v + mix first_v       to its slot of the V cache (first_v: the same token's values of an earlier layer)
// FP32 arithmetic, BF16 or FP32 storage. A group of G lanes owns one head of one row and keeps it in registers.
#include "dtype_io.cuh"
#include "host_util.h"

namespace ff {

constexpr int HN_THREADS = 256;

// NV: vectors of 8 elements a lane holds
template <typename T, int G, int NV>
__global__ void __launch_bounds__(HN_THREADS)
head_norm_kv_kernel(T* __restrict__ qkv, const int* __restrict__ slots, T* __restrict__ kcache, T* __restrict__ vcache,
                    const T* __restrict__ first_v, int rows, int hq, int hkv, int dim, int dk, int dv, int block_size, int num_blocks,
                    int ld, int ldf, float eps, float mix, const float* __restrict__ wq, const float* __restrict__ wk,
                    const float2* __restrict__ cos_sin, int half, int* status) {
  pdl_trigger();
  pdl_wait();
  const int heads = hq + 2 * hkv;
  const long long item = ((long long)blockIdx.x * HN_THREADS + threadIdx.x) / G;
  const int gl = threadIdx.x & (G - 1);
  const bool live = item < (long long)rows * heads;
  const int row = live ? (int)(item / heads) : 0, head = live ? (int)(item % heads) : 0;
  const bool is_q = head < hq, is_v = head >= hq + hkv;
  const int d = is_v ? dv : dk;
  T* base = qkv + (size_t)row * ld + (is_v ? (size_t)(hq + hkv) * dk + (size_t)(head - hq - hkv) * dv : (size_t)head * dk);
  float v[NV][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (gl + i * G) * 8;
    if (live && c < d) {
      load8(base + c, v[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(v[i][j], v[i][j], ss);
    }
  }
#pragma unroll
  for (int o = G / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o, G);
  if (!live) return;
  if (!is_v) {
    const float r = 1.0f / sqrtf(ss / (float)dim + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= r;
    const float* w = is_q ? wq : wk;
    if (w != nullptr) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (gl + i * G) * 8;
        if (c < d) {
          float f[8];
          load8(w + c, f);
#pragma unroll
          for (int j = 0; j < 8; ++j) v[i][j] *= f[j];
        }
      }
    }
    if (cos_sin != nullptr) {
      const float2* tab = cos_sin + (size_t)row * half;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int p = (gl + i * G) * 4;                    // first pair of this vector
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (p + j < half) {
            const float2 t = tab[p + j];
            const float a = v[i][2 * j], b = v[i][2 * j + 1];
            v[i][2 * j] = a * t.x - b * t.y;
            v[i][2 * j + 1] = b * t.x + a * t.y;
          }
      }
    }
  } else if (first_v != nullptr) {
    const T* fv = first_v + (size_t)row * ldf + (size_t)(head - hq - hkv) * dv;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (gl + i * G) * 8;
      if (c < d) {
        float f[8];
        load8(fv + c, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] = (1.0f - mix) * v[i][j] + mix * f[j];
      }
    }
  }
  T* dst = base;
  if (!is_q) {
    const int slot = slots[row];
    if (slot < 0) return;                                  // padding row: nothing cached
    const int blk = slot / block_size, off = slot - blk * block_size;
    const int kvh = is_v ? head - hq - hkv : head - hq;
    if (blk >= num_blocks) { if (gl == 0) set_status(status, KID_ROPE_KV, FF_ERR_BOUNDS, row, slot); return; }
    if (gl == 0) dbg_write_once(status, KID_ROPE_KV, is_v ? DBG_KV_V : DBG_KV_K, (long long)slot * hkv + kvh);
    dst = (is_v ? vcache : kcache) + (((size_t)blk * hkv + kvh) * block_size + off) * d;
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (gl + i * G) * 8;
    if (c < d) store8(dst + c, v[i]);
  }
}

template <typename T>
static int head_norm_launch(void* qkv, const int* slots, void* kcache, void* vcache, const void* first_v, int rows, int hq, int hkv, int dim,
                            int dk, int dv, int block_size, int num_blocks, int ld, int ldf, float eps, float mix, const float* wq, const float* wk,
                            const float2* cos_sin, int half, int* status, cudaStream_t s) {
  const int vecs = (dk > dv ? dk : dv) / 8;
  const long long items = (long long)rows * (hq + 2 * hkv);
  auto go = [&](auto kern, int g) -> int {
    const long long blocks = (items * g + HN_THREADS - 1) / HN_THREADS;
    if (int r = launch_pdl(kern, dim3((unsigned)blocks), dim3(HN_THREADS), 0, s, 0, (T*)qkv, slots, (T*)kcache, (T*)vcache, (const T*)first_v,
                           rows, hq, hkv, dim, dk, dv, block_size, num_blocks, ld, ldf, eps, mix, wq, wk, cos_sin, half, status)) return r;
    return launch_result();
  };
  if (vecs <= 8) return go(head_norm_kv_kernel<T, 8, 1>, 8);
  if (vecs <= 16) return go(head_norm_kv_kernel<T, 16, 1>, 16);
  if (vecs <= 32) return go(head_norm_kv_kernel<T, 32, 1>, 32);
  if (vecs <= 128) return go(head_norm_kv_kernel<T, 32, 4>, 32);
  return FF_HOST_TOO_LARGE;
}

}  // namespace ff
using namespace ff;

// wq, wk: FP32 norm weights of dk elements, or null; cos_sin: float2 [rows, half], or null
FF_EXPORT int ff_head_norm_kv(void* qkv, const int* slots, void* kcache, void* vcache, const void* first_v, int rows, int hq, int hkv,
                              int dim, int dk, int dv, int block_size, int num_blocks, int ld, int ldf, float eps, float mix,
                              const float* wq, const float* wk, const float* cos_sin, int half, int f32, int* status, cudaStream_t s) {
  if (rows <= 0 || hq <= 0 || hkv <= 0 || dim <= 0 || dk < dim || dk % 8 || dv <= 0 || dv % 8 || block_size <= 0) return FF_HOST_BAD_SHAPE;
  if (half < 0 || 2 * half > dim || (cos_sin != nullptr && half == 0)) return FF_HOST_BAD_SHAPE;
  if ((reinterpret_cast<uintptr_t>(wq) & 15) || (reinterpret_cast<uintptr_t>(wk) & 15)) return FF_HOST_BAD_ALIGN;
  const float2* cs = reinterpret_cast<const float2*>(cos_sin);
  if (ld % 8 || (first_v != nullptr && ldf % 8)) return FF_HOST_BAD_ALIGN;
  if (f32) return head_norm_launch<float>(qkv, slots, kcache, vcache, first_v, rows, hq, hkv, dim, dk, dv, block_size, num_blocks, ld, ldf, eps, mix, wq, wk, cs, half, status, s);
  return head_norm_launch<__nv_bfloat16>(qkv, slots, kcache, vcache, first_v, rows, hq, hkv, dim, dk, dv, block_size, num_blocks, ld, ldf, eps, mix, wq, wk, cs, half, status, s);
}
