// RMS norm of the queries and keys of packed projection rows, rotation, value blending, and the paged-cache write
// (rotate-half positions without a norm: rope_kv_paged in rope_act_sample.cu).
// head_norm_kv: norm per head, rotation of neighbouring elements
//   row = [hq query heads | hkv key heads | hkv value heads | ...], heads `dk` / `dv` elements apart of which the first
//   `dim` count for the norm (the rest is zero padding)
//   q <- rot(q / rms(q) * wq)            in the row         (weights and rotation where they are given: neighbours 2i, 2i + 1 of
//   k <- rot(k / rms(k) * wk)            to its slot         the first elements turn by the row's table of cosines and sines)
//                                        to its slot of the K cache [block][kv head][block_size][dk]
//   (q and k may also stay as they are: then q is not touched; v may be divided by its root mean square)
//   v <- (1 - mix) v + mix first_v       to its slot of the V cache (first_v: the same token's values of an earlier layer)
// FP32 arithmetic, BF16 or FP32 storage. A group of G lanes owns one head of one row and keeps it in registers.
// Optional query temperature: the query at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1).
// row_norm_kv: a block owns a row in shared memory; the norm runs over all q heads together and all k heads together (or per
// head), and rotated pairs are elements i and i + half (or neighbours).
// latent_norm_kv: latent attention. row = [... | rotated part of every query head | latent | rotated key part]; the cache row is
// [latent / rms(latent) * w | rotated key], the rotated query parts go behind the heads' latent queries.
#include "dtype_io.cuh"
#include "host_util.h"
#include <type_traits>

namespace ff {

constexpr int HN_THREADS = 256;

struct QueryTemp { const int* positions; float coef; int every; };
__device__ __forceinline__ float query_factor(const QueryTemp& t, int row) {
  if (t.positions == nullptr) return 1.0f;
  return 1.0f + t.coef * logf((float)((max(t.positions[row], 0) + 1) / t.every) + 1.0f);
}

// Which heads are normed: qk 0: q and k stay as they are; vdim > 0: values are divided by their root mean square over vdim elements.
struct HeadForm { int qk = 1, vdim = 0; };

// NV: vectors of 8 elements a lane holds
template <typename T, int G, int NV>
__global__ void __launch_bounds__(HN_THREADS)
head_norm_kv_kernel(T* __restrict__ qkv, const int* __restrict__ slots, T* __restrict__ kcache, T* __restrict__ vcache,
                    const T* __restrict__ first_v, int rows, int hq, int hkv, int dim, int dk, int dv, int block_size, int num_blocks,
                    int ld, int ldf, float eps, float mix, const float* __restrict__ wq, const float* __restrict__ wk,
                    const float2* __restrict__ cos_sin, int half, const QueryTemp temp, const HeadForm form, int* status) {
  pdl_trigger();
  pdl_wait();
  const int first = form.qk ? 0 : hq, heads = hq + 2 * hkv - first;
  const long long item = ((long long)blockIdx.x * HN_THREADS + threadIdx.x) / G;
  const int gl = threadIdx.x & (G - 1);
  const bool live = item < (long long)rows * heads;
  const int row = live ? (int)(item / heads) : 0, head = first + (live ? (int)(item % heads) : 0);
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
  if (is_v && form.vdim > 0) {
    const float r = 1.0f / sqrtf(ss / (float)form.vdim + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= r;
  }
  if (!is_v && form.qk) {
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
    if (is_q && temp.positions != nullptr) {
      const float f = query_factor(temp, row);
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] *= f;
    }
  } else if (is_v && first_v != nullptr) {
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
                            const float2* cos_sin, int half, const QueryTemp& temp, const HeadForm& form, int* status, cudaStream_t s) {
  const int vecs = (dk > dv ? dk : dv) / 8;
  const long long items = (long long)rows * ((form.qk ? hq : 0) + 2 * hkv);
  auto go = [&](auto kern, int g) -> int {
    const long long blocks = (items * g + HN_THREADS - 1) / HN_THREADS;
    if (int r = launch_pdl(kern, dim3((unsigned)blocks), dim3(HN_THREADS), 0, s, 0, (T*)qkv, slots, (T*)kcache, (T*)vcache, (const T*)first_v,
                           rows, hq, hkv, dim, dk, dv, block_size, num_blocks, ld, ldf, eps, mix, wq, wk, cos_sin, half, temp, form, status)) return r;
    return launch_result();
  };
  if (vecs <= 8) return go(head_norm_kv_kernel<T, 8, 1>, 8);
  if (vecs <= 16) return go(head_norm_kv_kernel<T, 16, 1>, 16);
  if (vecs <= 32) return go(head_norm_kv_kernel<T, 32, 1>, 32);
  if (vecs <= 128) return go(head_norm_kv_kernel<T, 32, 4>, 32);
  return FF_HOST_TOO_LARGE;
}

// What row_norm_kv adds: norms over whole projections (weights then cover all heads), pairs (i, i + half).
struct RowForm { int whole, halves; };

// VEC: halves turn and half is a multiple of 8
template <typename T, bool VEC>
__global__ void __launch_bounds__(HN_THREADS)
row_norm_kv_kernel(T* __restrict__ qkv, const int* __restrict__ slots, T* __restrict__ kcache, T* __restrict__ vcache, int hq, int hkv, int dim,
                   int dk, int dv, int block_size, int num_blocks, int ld, float eps, const float* __restrict__ wq, const float* __restrict__ wk,
                   const float2* __restrict__ cos_sin, int half, const RowForm form, const QueryTemp temp, int* status) {
  pdl_trigger();
  extern __shared__ __align__(16) float rk_row[];          // [(hq + hkv) * dk] the row, then one factor per head
  __shared__ float s_red[2][HN_THREADS / 32];
  const int row = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int heads = hq + hkv, nvec = heads * dk / 8, q_elems = hq * dk;
  float* s_r = rk_row + heads * dk;
  T* base = qkv + (size_t)row * ld;
  pdl_wait();
  float sq = 0.f, sk = 0.f;
  for (int i = tid; i < nvec; i += HN_THREADS) {
    float v[8];
    load8(base + i * 8, v);
    store8(rk_row + i * 8, v);
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(v[j], v[j], ss);
    if (i * 8 < q_elems) sq += ss; else sk += ss;
  }
  if (form.whole) {
    sq = warp_sum(sq); sk = warp_sum(sk);
    if (lane == 0) { s_red[0][warp] = sq; s_red[1][warp] = sk; }
    __syncthreads();
    sq = warp_sum(lane < HN_THREADS / 32 ? s_red[0][lane] : 0.f);
    sk = warp_sum(lane < HN_THREADS / 32 ? s_red[1][lane] : 0.f);
    const float rq = 1.0f / sqrtf(sq / (float)(hq * dim) + eps), rk = 1.0f / sqrtf(sk / (float)(max(hkv, 1) * dim) + eps);
    for (int h = tid; h < heads; h += HN_THREADS) s_r[h] = h < hq ? rq : rk;
  } else {
    __syncthreads();
    for (int h = warp; h < heads; h += HN_THREADS / 32) {
      float ss = 0.f;
      for (int c = lane; c < dk; c += 32) ss = fmaf(rk_row[h * dk + c], rk_row[h * dk + c], ss);
      ss = warp_sum(ss);
      if (lane == 0) s_r[h] = 1.0f / sqrtf(ss / (float)dim + eps);
    }
  }
  __syncthreads();
  const int slot = hkv > 0 ? slots[row] : -1;              // negative: padding row, nothing cached
  const int blk = slot / block_size, off = slot - blk * block_size;
  const bool cached = slot >= 0 && blk < num_blocks;
  if (slot >= 0 && !cached && tid == 0) set_status(status, KID_ROPE_KV, FF_ERR_BOUNDS, row, slot);
  const float tf = query_factor(temp, row);
  const float2* tab = cos_sin != nullptr ? cos_sin + (size_t)row * half : nullptr;
  const int dims = tab != nullptr ? 2 * half : 0, vph = dk / 8;
  for (int i = tid; i < nvec; i += HN_THREADS) {
    const int h = i / vph, c = (i - h * vph) * 8;
    const bool is_q = h < hq;
    if (!is_q && !cached) continue;
    const float* x = rk_row + h * dk;
    const float* w = is_q ? wq : wk;
    if (w != nullptr && form.whole) w += (is_q ? h : h - hq) * dk;
    const float r = s_r[h];
    float v[8];
    if (VEC) {                                             // a vector's partners are a vector
      float f[8];
      load8(x + c, v);
      if (w != nullptr) {
        load8(w + c, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] *= f[j];
      }
      if (c < dims) {
        const bool first = c < half;
        const int o = first ? c + half : c - half;
        float b[8];
        load8(x + o, b);
        if (w != nullptr) {
          load8(w + o, f);
#pragma unroll
          for (int j = 0; j < 8; ++j) b[j] *= f[j];
        }
        const float4* tp = reinterpret_cast<const float4*>(tab + (first ? c : o));
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
          const float4 t = tp[j >> 1];                     // (cos, sin) of two pairs
          v[j] = first ? v[j] * t.x - b[j] * t.y : v[j] * t.x + b[j] * t.y;
          v[j + 1] = first ? v[j + 1] * t.z - b[j + 1] * t.w : v[j + 1] * t.z + b[j + 1] * t.w;
        }
      }
      const float s = is_q ? r * tf : r;
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] *= s;
    } else
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int e = c + j;
      float a = x[e] * r * (w != nullptr ? w[e] : 1.0f);
      if (e < dims) {
        const bool first = form.halves ? e < half : (e & 1) == 0;
        const int o = form.halves ? (first ? e + half : e - half) : e ^ 1;
        const float2 t = tab[form.halves ? (first ? e : o) : e >> 1];
        const float b = x[o] * r * (w != nullptr ? w[o] : 1.0f);
        a = first ? a * t.x - b * t.y : a * t.x + b * t.y;
      }
      v[j] = is_q ? a * tf : a;
    }
    if (is_q) { store8(base + i * 8, v); continue; }
    if (c == 0) dbg_write_once(status, KID_ROPE_KV, DBG_KV_K, (long long)slot * hkv + h - hq);
    store8(kcache + (((size_t)blk * hkv + h - hq) * block_size + off) * dk + c, v);
  }
  if (!cached) return;
  const T* vals = base + (size_t)heads * dk;
  for (int i = tid; i < hkv * dv / 8; i += HN_THREADS) {
    const int h = i * 8 / dv, c = i * 8 - h * dv;
    float v[8];
    load8(vals + i * 8, v);
    if (c == 0) dbg_write_once(status, KID_ROPE_KV, DBG_KV_V, (long long)slot * hkv + h);
    store8(vcache + (((size_t)blk * hkv + h) * block_size + off) * dv + c, v);
  }
}

constexpr int LN_THREADS = 128;

template <typename T>
__global__ void __launch_bounds__(LN_THREADS)
latent_norm_kv_kernel(const T* __restrict__ p, const int* __restrict__ slots, T* __restrict__ cache, T* __restrict__ q_full, int heads, int rank,
                      int rank_pad, int rot_pad, int q_rot_col, int latent_col, int block_size, int num_blocks, int ld, float eps,
                      const float* __restrict__ w, const float2* __restrict__ cos_sin, int half, int* status) {
  pdl_trigger();
  __shared__ float s_red[LN_THREADS / 32];
  const int row = blockIdx.x, tid = threadIdx.x, width = rank_pad + rot_pad;
  pdl_wait();
  const T* base = p + (size_t)row * ld;
  const float2* tab = cos_sin + (size_t)row * half;
  auto turn = [&](float (&v)[8], int c) {                  // neighbours from element c on
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = (c >> 1) + j;
      if (i < half) {
        const float2 t = tab[i];
        const float a = v[2 * j], b = v[2 * j + 1];
        v[2 * j] = a * t.x - b * t.y;
        v[2 * j + 1] = b * t.x + a * t.y;
      }
    }
  };
  const int rvec = rot_pad / 8;
  for (int i = tid; i < heads * rvec; i += LN_THREADS) {
    const int h = i / rvec, c = (i - h * rvec) * 8;
    float v[8];
    load8(base + q_rot_col + i * 8, v);
    turn(v, c);
    store8(q_full + ((size_t)row * heads + h) * width + rank_pad + c, v);
  }
  const int slot = slots[row];
  if (slot < 0) return;                                    // padding row: nothing cached
  const int blk = slot / block_size;
  if (blk >= num_blocks) { if (tid == 0) set_status(status, KID_MLA, FF_ERR_BOUNDS, row, slot); return; }
  const T* lat = base + latent_col;
  T* dst = cache + (size_t)slot * width;
  float ss = 0.f;
  for (int i = tid; i < rank_pad / 8; i += LN_THREADS) {
    float v[8];
    load8(lat + i * 8, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(v[j], v[j], ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) s_red[tid >> 5] = ss;
  __syncthreads();
  const float r = 1.0f / sqrtf(warp_sum((tid & 31) < LN_THREADS / 32 ? s_red[tid & 31] : 0.f) / (float)rank + eps);
  for (int i = tid; i < rank_pad / 8; i += LN_THREADS) {
    float v[8], f[8];
    load8(lat + i * 8, v);
    load8(w + i * 8, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = v[j] * r * f[j];
    store8(dst + i * 8, v);
  }
  for (int i = tid; i < rvec; i += LN_THREADS) {
    float v[8];
    load8(lat + rank_pad + i * 8, v);
    turn(v, i * 8);
    store8(dst + rank_pad + i * 8, v);
  }
  if (tid == 0) dbg_write_once(status, KID_MLA, DBG_KV_K, slot);
}

template <typename T>
static int row_norm_launch(void* qkv, const int* slots, void* kcache, void* vcache, int rows, int hq, int hkv, int dim, int dk, int dv, int block_size,
                           int num_blocks, int ld, float eps, const float* wq, const float* wk, const float2* cos_sin, int half, const RowForm& form,
                           const QueryTemp& temp, int* status, cudaStream_t s) {
  const int smem = ((hq + hkv) * dk + hq + hkv) * 4;
  if (smem > 200 * 1024) return FF_HOST_TOO_LARGE;
  const bool vec = (cos_sin == nullptr || (form.halves && half % 8 == 0)) && ((reinterpret_cast<uintptr_t>(wq) | reinterpret_cast<uintptr_t>(wk)) & 15) == 0;
  auto kern = vec ? row_norm_kv_kernel<T, true> : row_norm_kv_kernel<T, false>;
  if (int r = opt_in_smem(kern, smem)) return r;
  if (int r = launch_pdl(kern, dim3(rows), dim3(HN_THREADS), smem, s, 0, (T*)qkv, slots, (T*)kcache, (T*)vcache, hq, hkv, dim, dk, dv, block_size,
                         num_blocks, ld, eps, wq, wk, cos_sin, half, form, temp, status)) return r;
  return launch_result();
}

}  // namespace ff
using namespace ff;

// As ff_head_norm_kv without value blending. whole: q and k are normed over all their heads (wq [hq * dk], wk [hkv * dk]), otherwise
// per head (wq, wk [dk]); halves: elements i and i + half turn together, otherwise neighbours. hkv = 0: queries only.
FF_EXPORT int ff_row_norm_kv(void* qkv, const int* slots, void* kcache, void* vcache, int rows, int hq, int hkv, int dim, int dk, int dv,
                             int block_size, int num_blocks, int ld, float eps, const float* wq, const float* wk, const float* cos_sin, int half,
                             int whole, int halves, const int* positions, float coef, int every, int f32, int* status, cudaStream_t s) {
  if (rows <= 0 || hq <= 0 || hkv < 0 || dim <= 0 || dk < dim || dk % 8 || dv < 0 || dv % 8 || block_size <= 0) return FF_HOST_BAD_SHAPE;
  if (half < 0 || 2 * half > dim || (cos_sin != nullptr && half == 0) || (positions != nullptr && every < 1)) return FF_HOST_BAD_SHAPE;
  if (hkv > 0 && (slots == nullptr || kcache == nullptr || vcache == nullptr || dv == 0)) return FF_HOST_BAD_SHAPE;
  if (ld % 8) return FF_HOST_BAD_ALIGN;
  const float2* cs = reinterpret_cast<const float2*>(cos_sin);
  const RowForm form = {whole, halves};
  const QueryTemp temp = {positions, coef, every};
  if (f32) return row_norm_launch<float>(qkv, slots, kcache, vcache, rows, hq, hkv, dim, dk, dv, block_size, num_blocks, ld, eps, wq, wk, cs, half, form, temp, status, s);
  return row_norm_launch<__nv_bfloat16>(qkv, slots, kcache, vcache, rows, hq, hkv, dim, dk, dv, block_size, num_blocks, ld, eps, wq, wk, cs, half, form, temp, status, s);
}

// p: packed rows with the rotated query parts [heads, rot_pad] at column q_rot_col and [latent (rank_pad) | key (rot_pad)] at
// latent_col; cache [blocks, 1, block_size, rank_pad + rot_pad]; q_full [rows, heads, rank_pad + rot_pad] (its last rot_pad columns
// are written); w FP32 [rank_pad]; cos_sin float2 [rows, half].
FF_EXPORT int ff_latent_norm_kv(const void* p, const int* slots, void* cache, void* q_full, int rows, int heads, int rank, int rank_pad, int rot_pad,
                                int q_rot_col, int latent_col, int block_size, int num_blocks, int ld, float eps, const float* w,
                                const float* cos_sin, int half, int f32, int* status, cudaStream_t s) {
  if (rows <= 0 || heads <= 0 || rank <= 0 || rank_pad < rank || rank_pad % 8 || rot_pad % 8 || half <= 0 || 2 * half > rot_pad || block_size <= 0)
    return FF_HOST_BAD_SHAPE;
  if (ld % 8 || q_rot_col % 8 || latent_col % 8 || (reinterpret_cast<uintptr_t>(w) & 15)) return FF_HOST_BAD_ALIGN;
  const float2* cs = reinterpret_cast<const float2*>(cos_sin);
  auto go = [&](auto kern, auto* t) -> int {
    using T = std::remove_pointer_t<decltype(t)>;
    if (int r = launch_pdl(kern, dim3(rows), dim3(LN_THREADS), 0, s, 0, (const T*)p, slots, (T*)cache, (T*)q_full, heads, rank, rank_pad, rot_pad,
                           q_rot_col, latent_col, block_size, num_blocks, ld, eps, w, cs, half, status)) return r;
    return launch_result();
  };
  if (f32) return go(latent_norm_kv_kernel<float>, (float*)nullptr);
  return go(latent_norm_kv_kernel<__nv_bfloat16>, (__nv_bfloat16*)nullptr);
}

// wq, wk: FP32 norm weights of dk elements, or null; cos_sin: float2 [rows, half], or null; positions: query temperature, or null;
// hkv = 0: queries only; norm_qk, v_norm_dim: HeadForm
FF_EXPORT int ff_head_norm_kv(void* qkv, const int* slots, void* kcache, void* vcache, const void* first_v, int rows, int hq, int hkv,
                              int dim, int dk, int dv, int block_size, int num_blocks, int ld, int ldf, float eps, float mix,
                              const float* wq, const float* wk, const float* cos_sin, int half, const int* positions, float coef,
                              int every, int norm_qk, int v_norm_dim, int f32, int* status, cudaStream_t s) {
  if (!norm_qk && (hkv == 0 || wq != nullptr || wk != nullptr || cos_sin != nullptr || positions != nullptr)) return FF_HOST_UNSUPPORTED;
  if (v_norm_dim < 0 || v_norm_dim > dv) return FF_HOST_BAD_SHAPE;
  const HeadForm form = {norm_qk, v_norm_dim};
  if (rows <= 0 || hq <= 0 || hkv < 0 || (positions != nullptr && every < 1) || dim <= 0 || dk < dim || dk % 8 || dv <= 0 || dv % 8 || block_size <= 0) return FF_HOST_BAD_SHAPE;
  if (half < 0 || 2 * half > dim || (cos_sin != nullptr && half == 0)) return FF_HOST_BAD_SHAPE;
  if ((reinterpret_cast<uintptr_t>(wq) & 15) || (reinterpret_cast<uintptr_t>(wk) & 15)) return FF_HOST_BAD_ALIGN;
  const float2* cs = reinterpret_cast<const float2*>(cos_sin);
  const QueryTemp temp = {positions, coef, every};
  if (ld % 8 || (first_v != nullptr && ldf % 8)) return FF_HOST_BAD_ALIGN;
  if (f32) return head_norm_launch<float>(qkv, slots, kcache, vcache, first_v, rows, hq, hkv, dim, dk, dv, block_size, num_blocks, ld, ldf, eps, mix, wq, wk, cs, half, temp, form, status, s);
  return head_norm_launch<__nv_bfloat16>(qkv, slots, kcache, vcache, first_v, rows, hq, hkv, dim, dk, dv, block_size, num_blocks, ld, ldf, eps, mix, wq, wk, cs, half, temp, form, status, s);
}
