// Windowed attention whose heads' weights are mixed before they meet the values (talk_simt.cu) on tensor cores: BF16, heads of up to 128
// elements, paged cache with 64-token pages.
//   w_g(i, j) = 2^(s_g(i, j) - z_g(i)),  z_g(i) the logarithm of the soft-max's denominator      M_h = sum_g talk[h, g] w_g      o_h = M_h v
// The mixed weights of a head need the normalised weights of every head, so no head can run its soft-max and its value product in one
// pass. Prompts take three:
//   1. attn_prefill_tc (attention_tc.cu) leaves z of every row and head;
//   2. talk_weights : 16 query rows and all heads per CTA, 32 keys at a time: scores again, weights in FP16 through shared memory, the
//      product with the mixing matrix (heads as its inner dimension), mixed weights in BF16 to scratch;
//   3. talk_values  : scratch times values, 64 query rows of up to four heads that share a value head per CTA.
// 2 and 3 go over the prompt in rounds whose scratch stays in the L2 cache. Decoded tokens take two and a merge:
//   talk_scores : scores of a key / value head's query heads over a range of pages, in FP32, and their maximum and sum;
//   talk_decode : the weights of all heads for a page, mixed for the heads of one value head (the accumulators of that product are the
//                 operand of the next), times the values.
#include "host_util.h"
#include "mma_sync.cuh"
#include <cuda_fp16.h>

namespace ff {

constexpr int TK_PAGE = 64;
constexpr float TK_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void tk_cp16(void* dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory"); }
__device__ __forceinline__ void tk_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void tk_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ float tk_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ uint32_t pack_half2(float x, float y) { const __half2 h = __floats2half2_rn(x, y); return *reinterpret_cast<const uint32_t*>(&h); }
__device__ __forceinline__ void mma_f16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct TalkArgs {
  const __nv_bfloat16* q; const __nv_bfloat16* kcache; const __nv_bfloat16* vcache;
  const int* block_table; const int* q_start; const int* q_lens; const int* ctx_lens;
  const float* talk; const float* z;         // z: [rows, H], base 2 (prompts)
  __nv_bfloat16* out; __nv_bfloat16* scratch;
  int H, G, dk, dv, ldq, ldo, max_blocks, num_blocks, window, band;      // band: pages a tile's rows see at most
  int tile0, tiles;                          // this round's tiles of 64 rows
  int parts;                                 // CTAs that share the keys of 16 rows (talk_weights)
  float scale_log2;
  int* status;
};

// pages and positions of a 64-row tile
struct TalkTile {
  int real, first, lo_page, hi_page;         // rows, position of row 0
  __device__ TalkTile(const TalkArgs& p, int b, int tile) {
    const int qlen = p.q_lens[b], past = p.ctx_lens[b] - qlen, r0 = tile * 64;
    real = min(64, qlen - r0);
    first = past + r0;
    lo_page = max(0, first - p.window + 1) / TK_PAGE;
    hi_page = (first + max(real, 1) - 1) / TK_PAGE;
  }
};

// a fragment of the mixing matrix: 16 heads from row0 (rows past `rows` of them and columns past H are zero), 16 columns from col0
__device__ __forceinline__ void talk_frag(const float* talk, int H, int row0, int rows, int col0, int lane, uint32_t (&a)[4]) {
  const int g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = g + 8 * (i & 1), c = col0 + 2 * t + 8 * (i >> 1);
    const bool on = r < rows && row0 + r < H;
    a[i] = pack_half2(on && c < H ? talk[(size_t)(row0 + r) * H + c] : 0.f, on && c + 1 < H ? talk[(size_t)(row0 + r) * H + c + 1] : 0.f);
  }
}

// ---------------------------------------------------------------------------------------
// talk_weights: grid (4 * tiles, parts, sequences), 256 threads. KP: key width padded to 64 or 128; HB: blocks of 16 heads; NB: query heads
// of one key head that a warp takes together
// ---------------------------------------------------------------------------------------
constexpr int TW_KEYS = 32;
__device__ __forceinline__ uint32_t tw_off(int h, int chunk) {        // byte offset of 16-byte chunk 0..63 of head h's 16 x 32 weights
  return (uint32_t)(h * 1024 + ((chunk & ~7) | ((chunk ^ ((chunk >> 3) & 3) ^ h) & 7)) * 16);
}

template <int KP, int HB, int NB>
__global__ void __launch_bounds__(256, 1)
talk_weights_kernel(const TalkArgs p) {
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t tk_raw[];
  constexpr int KCH = KP / 8, QB = 16 * KP * 2, KB = TW_KEYS * KP * 2;
  uint8_t* sQ = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tk_raw) + 127) & ~uintptr_t(127));
  uint8_t* sK = sQ + p.H * QB;                             // [G][32 keys]
  uint8_t* sP = sK + p.G * KB;                             // [16 HB][16 x 32]
  float* sZ = reinterpret_cast<float*>(sP + HB * 16 * 1024);           // [H][16]
  pdl_wait();
  const int b = blockIdx.z, tile = p.tile0 + (blockIdx.x >> 2), sub = blockIdx.x & 3, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, tq = lane & 3, H = p.H, G = p.G, per = H / G;
  const TalkTile tl(p, b, tile);
  const int rows = min(16, tl.real - sub * 16);
  if (rows <= 0) return;
  const int row0 = p.q_start[b] + tile * 64 + sub * 16, pos0 = tl.first + sub * 16;
  const int bandw = p.band * TK_PAGE, keys = (tl.hi_page - tl.lo_page + 1) * TK_PAGE, base = tl.lo_page * TK_PAGE;
  __nv_bfloat16* dst = p.scratch + ((((size_t)b * p.tiles + (blockIdx.x >> 2)) * H) * 64 + sub * 16) * bandw;
  // visible steps of 32 keys; the first part writes the zeros of the others
  const int v0 = max(0, pos0 - p.window + 1 - base) / TW_KEYS, v1 = min(keys, pos0 + rows - base + TW_KEYS - 1) / TW_KEYS;
  if (blockIdx.y == 0)
    for (int step = 0; step < keys / TW_KEYS; ++step)
      if (step < v0 || step >= v1)
        for (int i = tid; i < H * 64; i += 256)
          *reinterpret_cast<uint4*>(dst + ((size_t)(i >> 6) * 64 + ((i >> 2) & 15)) * bandw + step * TW_KEYS + (i & 3) * 8) = make_uint4(0, 0, 0, 0);
  const int ka = v0 + (v1 - v0) * (int)blockIdx.y / p.parts, kb = v0 + (v1 - v0) * ((int)blockIdx.y + 1) / p.parts;
  if (ka >= kb) return;
  for (int i = tid; i < H * 16 * KCH; i += 256) {
    const int h = i / (16 * KCH), r = (i / KCH) & 15, c = i % KCH;
    uint8_t* at = sQ + h * QB + ms_off(r, c, KCH);
    if (r < rows && c * 8 < p.dk) tk_cp16(at, p.q + (size_t)(row0 + r) * p.ldq + (size_t)h * p.dk + c * 8);
    else *reinterpret_cast<uint4*>(at) = make_uint4(0, 0, 0, 0);
  }
  for (int i = tid; i < H * 16; i += 256) { const int h = i >> 4, r = i & 15; sZ[i] = r < rows ? p.z[(size_t)(row0 + r) * H + h] : 0.f; }
  for (int i = tid; i < HB * 16 * 1024 / 16; i += 256) reinterpret_cast<uint4*>(sP)[i] = make_uint4(0, 0, 0, 0);       // rows past H stay zero
  auto fetch = [&](int step) {
    const int k0 = base + step * TW_KEYS;
    int blk = p.block_table[(size_t)b * p.max_blocks + k0 / TK_PAGE];
    const bool ok = blk >= 0 && blk < p.num_blocks;
    if (!ok) { if (tid == 0) set_status(p.status, KID_ATTN_PREFILL, FF_ERR_BOUNDS, b, k0); blk = 0; }
    for (int i = tid; i < G * TW_KEYS * KCH; i += 256) {
      const int g = i / (TW_KEYS * KCH), r = (i / KCH) & (TW_KEYS - 1), c = i % KCH;
      uint8_t* at = sK + g * KB + ms_off(r, c, KCH);
      if (c * 8 < p.dk) tk_cp16(at, p.kcache + (((size_t)blk * G + g) * TK_PAGE + k0 % TK_PAGE + r) * p.dk + c * 8);
      else *reinterpret_cast<uint4*>(at) = make_uint4(0, 0, 0, 0);
    }
  };
  fetch(ka);
  tk_commit();
  uint32_t tf[HB][HB][4];
#pragma unroll
  for (int i = 0; i < HB; ++i)
#pragma unroll
    for (int j = 0; j < HB; ++j) talk_frag(p.talk, H, 16 * i, 16, 16 * j, lane, tf[i][j]);
  const int batches = (per + NB - 1) / NB, ksteps = p.dk / 16;
  for (int step = ka; step < kb; ++step) {
    tk_wait<0>();
    __syncthreads();
    const int k0 = base + step * TW_KEYS;
    // ---- scores and weights
    for (int unit = warp; unit < G * batches; unit += 8) {
      const int g = unit / batches, h0 = g * per + (unit - g * batches) * NB, last = (g + 1) * per - 1;
      float s[NB][4][4];
#pragma unroll
      for (int n = 0; n < NB; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) s[n][i][0] = s[n][i][1] = s[n][i][2] = s[n][i][3] = 0.f;
      const uint32_t ak = smem_u32(sK + g * KB);
#pragma unroll 2
      for (int ks = 0; ks < ksteps; ++ks) {
        uint32_t bf[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
          ms_ldsm4(ak + ms_off(16 * j + ((lane >> 4) << 3) + (lane & 7), 2 * ks + ((lane >> 3) & 1), KCH), bf[j][0], bf[j][1], bf[j][2], bf[j][3]);
#pragma unroll
        for (int n = 0; n < NB; ++n) {
          uint32_t a[4];
          ms_ldsm4(smem_u32(sQ + min(h0 + n, last) * QB) + ms_off((lane & 7) + (((lane >> 3) & 1) << 3), 2 * ks + (lane >> 4), KCH), a[0], a[1], a[2], a[3]);
#pragma unroll
          for (int j = 0; j < 2; ++j) { ms_mma(s[n][2 * j], a, bf[j][0], bf[j][1]); ms_mma(s[n][2 * j + 1], a, bf[j][2], bf[j][3]); }
        }
      }
      const bool inside = k0 + TW_KEYS - 1 <= pos0 && k0 > pos0 + 15 - p.window;
#pragma unroll
      for (int n = 0; n < NB; ++n) {
        const int h = h0 + n;
        if (h > last) continue;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = gq + 8 * e, pos = pos0 + r;
          const float z = sZ[h * 16 + r];
          uint32_t w[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int key = k0 + 8 * i + 2 * tq;
            float x = tk_ex2(fmaf(s[n][i][2 * e], p.scale_log2, -z)), y = tk_ex2(fmaf(s[n][i][2 * e + 1], p.scale_log2, -z));
            if (!inside) {
              x = key <= pos && key > pos - p.window ? x : 0.f;
              y = key + 1 <= pos && key + 1 > pos - p.window ? y : 0.f;
            }
            w[i] = pack_half2(x, y);
          }
          // keys 8 i + 2 t + {0, 1} of row r: chunk 4 r + t
          *reinterpret_cast<uint4*>(sP + tw_off(h, 4 * r + tq)) = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
    }
    __syncthreads();
    if (step + 1 < kb) fetch(step + 1);
    tk_commit();
    // ---- mixed: a warp takes two rows; column n of chunk 4 r + c is key 8 (n / 2) + 2 c + n % 2, so a thread gets keys 8 t .. 8 t + 7
    const uint32_t ap = smem_u32(sP);
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      const int r = 2 * warp + rr;
      uint32_t bf[HB][2][4];
#pragma unroll
      for (int j = 0; j < HB; ++j)
#pragma unroll
        for (int c = 0; c < 2; ++c)
          ms_ldsm4t(ap + tw_off(16 * j + (lane & 7) + (((lane >> 3) & 1) << 3), 4 * r + 2 * c + (lane >> 4)), bf[j][c][0], bf[j][c][1], bf[j][c][2], bf[j][c][3]);
#pragma unroll
      for (int i = 0; i < HB; ++i) {
        float m[4][4];
#pragma unroll
        for (int c = 0; c < 4; ++c) m[c][0] = m[c][1] = m[c][2] = m[c][3] = 0.f;
#pragma unroll
        for (int j = 0; j < HB; ++j)
#pragma unroll
          for (int c = 0; c < 2; ++c) { mma_f16(m[2 * c], tf[i][j], bf[j][c][0], bf[j][c][1]); mma_f16(m[2 * c + 1], tf[i][j], bf[j][c][2], bf[j][c][3]); }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int h = 16 * i + gq + 8 * e;
          if (h < H)
            *reinterpret_cast<uint4*>(dst + ((size_t)h * 64 + r) * bandw + step * TW_KEYS + 8 * tq) =
                make_uint4(pack_bf16x2(m[0][2 * e], m[0][2 * e + 1]), pack_bf16x2(m[1][2 * e], m[1][2 * e + 1]), pack_bf16x2(m[2][2 * e], m[2][2 * e + 1]),
                           pack_bf16x2(m[3][2 * e], m[3][2 * e + 1]));
        }
      }
    }
  }
}

// ---------------------------------------------------------------------------------------
// talk_values: grid (tiles, G * batches of NH heads, sequences), 64 NH threads: a warp owns 32 rows of a head. DV: value width padded to
// 64 or 128
// ---------------------------------------------------------------------------------------
template <int DV, int NH>
__global__ void __launch_bounds__(64 * NH)
talk_values_kernel(const TalkArgs p) {
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t tk_raw[];
  constexpr int THREADS = 64 * NH, MB = NH * 64 * 128, VB = TK_PAGE * DV * 2, VCH = DV / 8;
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tk_raw) + 127) & ~uintptr_t(127));     // two of [weights | values]
  pdl_wait();
  const int b = blockIdx.z, tile = p.tile0 + blockIdx.x, per = p.H / p.G, batches = (per + NH - 1) / NH;
  const int g = blockIdx.y / batches, h0 = g * per + (blockIdx.y % batches) * NH, heads = min(NH, (g + 1) * per - h0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
  const TalkTile tl(p, b, tile);
  if (tl.real <= 0) return;
  const int bandw = p.band * TK_PAGE, pages = tl.hi_page - tl.lo_page + 1;
  const __nv_bfloat16* src = p.scratch + (((size_t)b * p.tiles + blockIdx.x) * p.H + h0) * 64 * bandw;
  auto fetch = [&](int page) {
    uint8_t* m = sm + (page & 1) * (MB + VB);
    uint8_t* v = m + MB;
    for (int i = tid; i < heads * 64 * 8; i += THREADS) {
      const int r = i >> 3, c = i & 7;                     // rows past the prompt: never written, their products are not stored
      tk_cp16(m + ms_off(r, c, 8), src + (size_t)r * bandw + page * TK_PAGE + c * 8);
    }
    int blk = p.block_table[(size_t)b * p.max_blocks + tl.lo_page + page];
    if (blk < 0 || blk >= p.num_blocks) { if (tid == 0) set_status(p.status, KID_ATTN_PREFILL, FF_ERR_BOUNDS, b, page); blk = 0; }
    const __nv_bfloat16* vp = p.vcache + ((size_t)blk * p.G + g) * TK_PAGE * p.dv;
    for (int i = tid; i < TK_PAGE * VCH; i += THREADS) {
      const int r = i / VCH, c = i - r * VCH;
      if (c * 8 < p.dv) tk_cp16(v + ms_off(r, c, VCH), vp + (size_t)r * p.dv + c * 8);
      else *reinterpret_cast<uint4*>(v + ms_off(r, c, VCH)) = make_uint4(0, 0, 0, 0);
    }
  };
  float o[2][DV / 8][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) o[i][n][0] = o[i][n][1] = o[i][n][2] = o[i][n][3] = 0.f;
  fetch(0);
  tk_commit();
  const bool on = warp / 2 < heads;
  for (int page = 0; page < pages; ++page) {
    if (page + 1 < pages) fetch(page + 1);
    tk_commit();
    tk_wait<1>();
    __syncthreads();
    const uint32_t am = smem_u32(sm + (page & 1) * (MB + VB)), av = am + MB;
    if (on) {
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        uint32_t a[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i)
          ms_ldsm4(am + ms_off(warp * 32 + 16 * i + (lane & 7) + (((lane >> 3) & 1) << 3), 2 * ks + (lane >> 4), 8), a[i][0], a[i][1], a[i][2], a[i][3]);
#pragma unroll
        for (int np = 0; np < DV / 16; ++np) {
          uint32_t b0, b1, b2, b3;
          ms_ldsm4t(av + ms_off(ks * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), 2 * np + (lane >> 4), VCH), b0, b1, b2, b3);
#pragma unroll
          for (int i = 0; i < 2; ++i) { ms_mma(o[i][2 * np], a[i], b0, b1); ms_mma(o[i][2 * np + 1], a[i], b2, b3); }
        }
      }
    }
    __syncthreads();
  }
  if (!on) return;
  const int h = h0 + warp / 2;
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = (warp & 1) * 32 + 16 * i + gq + 8 * e;
      if (r >= tl.real) continue;
      __nv_bfloat16* orow = p.out + (size_t)(p.q_start[b] + tile * 64 + r) * p.ldo + (size_t)h * p.dv;
#pragma unroll
      for (int n = 0; n < DV / 8; ++n)
        if (8 * n + 2 * tq < p.dv) *reinterpret_cast<uint32_t*>(orow + 8 * n + 2 * tq) = pack_bf16x2(o[i][n][2 * e], o[i][n][2 * e + 1]);
    }
}

// ---------------------------------------------------------------------------------------
// decode: one row per sequence. scores FP32 [sequence, H, band * 64] (base 2, scaled), ml [sequence, splits, H] (maximum, sum)
// ---------------------------------------------------------------------------------------
struct TalkDecodeArgs {
  const __nv_bfloat16* q; const __nv_bfloat16* kcache; const __nv_bfloat16* vcache;
  const int* block_table; const int* ctx_lens; const float* talk;
  __nv_bfloat16* out; float* scores; float2* ml; float* part;          // part: [sequence, splits, H, dv], with more than one split
  int H, G, dk, dv, ldq, ldo, max_blocks, num_blocks, window, band, splits;
  float scale_log2, one;
  int* status;
};

struct TalkSpan {
  int ctx, lo_page, page, end;               // this split's pages page .. end - 1, counted from lo_page
  __device__ TalkSpan(const TalkDecodeArgs& p, int b, int split) {
    ctx = p.ctx_lens[b];
    lo_page = max(0, ctx - p.window) / TK_PAGE;
    const int pages = ctx > 0 ? (ctx - 1) / TK_PAGE - lo_page + 1 : 0, each = (pages + p.splits - 1) / p.splits;
    page = min(pages, split * each);
    end = min(pages, page + each);
  }
};

// grid (splits, G, sequences), 128 threads: 16 keys of a page per warp, the query heads of a key head as the rows of one 16-row tile
template <int KP>
__global__ void __launch_bounds__(128)
talk_scores_kernel(const TalkDecodeArgs p) {
  pdl_trigger();
  constexpr int KCH = KP / 8, KB = TK_PAGE * KP * 2;
  __shared__ __align__(128) uint8_t sQ[16 * KP * 2];
  __shared__ float s_red[4][16][2];
  extern __shared__ __align__(128) uint8_t tk_raw[];
  uint8_t* sK = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tk_raw) + 127) & ~uintptr_t(127));
  pdl_wait();
  const int split = blockIdx.x, g = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
  const int per = p.H / p.G;
  const TalkSpan sp(p, b, split);
  auto fetch = [&](int page) {
    int blk = p.block_table[(size_t)b * p.max_blocks + sp.lo_page + page];
    if (blk < 0 || blk >= p.num_blocks) { if (tid == 0) set_status(p.status, KID_ATTN_DECODE, FF_ERR_BOUNDS, b, page); blk = 0; }
    const __nv_bfloat16* kp = p.kcache + ((size_t)blk * p.G + g) * TK_PAGE * p.dk;
    uint8_t* k = sK + (page & 1) * KB;
    for (int i = tid; i < TK_PAGE * KCH; i += 128) {
      const int r = i / KCH, c = i - r * KCH;
      if (c * 8 < p.dk) tk_cp16(k + ms_off(r, c, KCH), kp + (size_t)r * p.dk + c * 8);
      else *reinterpret_cast<uint4*>(k + ms_off(r, c, KCH)) = make_uint4(0, 0, 0, 0);
    }
  };
  if (sp.page < sp.end) fetch(sp.page);
  tk_commit();
  for (int i = tid; i < 16 * KCH; i += 128) {
    const int r = i / KCH, c = i - r * KCH;
    *reinterpret_cast<uint4*>(sQ + ms_off(r, c, KCH)) =
        r < per && c * 8 < p.dk ? *reinterpret_cast<const uint4*>(p.q + (size_t)b * p.ldq + (size_t)(g * per + r) * p.dk + c * 8) : make_uint4(0, 0, 0, 0);
  }
  float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};
  const uint32_t aq = smem_u32(sQ);
  for (int page = sp.page; page < sp.end; ++page) {
    if (page + 1 < sp.end) fetch(page + 1);
    tk_commit();
    tk_wait<1>();
    __syncthreads();
    const uint32_t ak = smem_u32(sK + (page & 1) * KB);
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int ks = 0; ks < KP / 16; ++ks) {
      if (ks * 16 >= p.dk) break;
      uint32_t a[4], b0, b1, b2, b3;
      ms_ldsm4(aq + ms_off((lane & 7) + (((lane >> 3) & 1) << 3), 2 * ks + (lane >> 4), KCH), a[0], a[1], a[2], a[3]);
      ms_ldsm4(ak + ms_off(16 * warp + ((lane >> 4) << 3) + (lane & 7), 2 * ks + ((lane >> 3) & 1), KCH), b0, b1, b2, b3);
      ms_mma(s[0], a, b0, b1);
      ms_mma(s[1], a, b2, b3);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = gq + 8 * e;
      float m = mx[e];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int key = (sp.lo_page + page) * TK_PAGE + 16 * warp + 8 * i + 2 * tq + j;
          s[i][2 * e + j] = key < sp.ctx && key >= sp.ctx - p.window ? s[i][2 * e + j] * p.scale_log2 : -INFINITY;
          m = fmaxf(m, s[i][2 * e + j]);
        }
      if (m > -INFINITY) {
        sum[e] *= tk_ex2(mx[e] - m);
#pragma unroll
        for (int i = 0; i < 2; ++i) sum[e] += tk_ex2(s[i][2 * e] - m) + tk_ex2(s[i][2 * e + 1] - m);
      }
      mx[e] = m;
      if (r < per) {
        float* dst = p.scores + ((size_t)b * p.H + g * per + r) * p.band * TK_PAGE + page * TK_PAGE + 16 * warp + 2 * tq;
#pragma unroll
        for (int i = 0; i < 2; ++i) *reinterpret_cast<float2*>(dst + 8 * i) = make_float2(s[i][2 * e], s[i][2 * e + 1]);
      }
    }
    __syncthreads();
  }
  auto join = [](float& m, float& l, float om, float ol) {
    const float n = fmaxf(m, om);
    if (n > -INFINITY) l = l * tk_ex2(m - n) + ol * tk_ex2(om - n);
    m = n;
  };
#pragma unroll
  for (int e = 0; e < 2; ++e) {
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) join(mx[e], sum[e], __shfl_xor_sync(0xffffffffu, mx[e], o), __shfl_xor_sync(0xffffffffu, sum[e], o));
    if (tq == 0) { s_red[warp][gq + 8 * e][0] = mx[e]; s_red[warp][gq + 8 * e][1] = sum[e]; }
  }
  __syncthreads();
  if (tid < per) {
    float m = -INFINITY, l = 0.f;
    for (int w = 0; w < 4; ++w) join(m, l, s_red[w][tid][0], s_red[w][tid][1]);
    p.ml[((size_t)b * p.splits + split) * p.H + g * per + tid] = make_float2(m, l);
  }
}

// grid (splits, G, sequences), 128 threads
template <int DV, int HB>
__global__ void __launch_bounds__(128)
talk_decode_kernel(const TalkDecodeArgs p) {
  pdl_trigger();
  constexpr int VCH = DV / 8, VB = TK_PAGE * DV * 2;
  __shared__ __align__(128) uint8_t sP[HB * 16 * 128];     // [heads][64 keys], FP16
  __shared__ float s_z[HB * 16];
  extern __shared__ __align__(128) uint8_t tk_raw[];
  uint8_t* sV = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tk_raw) + 127) & ~uintptr_t(127));     // two pages, then [4][16][DV] sums
  pdl_wait();
  const int split = blockIdx.x, g = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
  const int per = p.H / p.G, H = p.H;
  const TalkSpan sp(p, b, split);
  auto fetch = [&](int page) {
    int blk = p.block_table[(size_t)b * p.max_blocks + sp.lo_page + page];
    if (blk < 0 || blk >= p.num_blocks) blk = 0;           // reported by talk_scores
    const __nv_bfloat16* vp = p.vcache + ((size_t)blk * p.G + g) * TK_PAGE * p.dv;
    uint8_t* v = sV + (page & 1) * VB;
    for (int i = tid; i < TK_PAGE * VCH; i += 128) {
      const int r = i / VCH, c = i - r * VCH;
      if (c * 8 < p.dv) tk_cp16(v + ms_off(r, c, VCH), vp + (size_t)r * p.dv + c * 8);
      else *reinterpret_cast<uint4*>(v + ms_off(r, c, VCH)) = make_uint4(0, 0, 0, 0);
    }
  };
  if (sp.page < sp.end) fetch(sp.page);
  tk_commit();
  for (int h = tid; h < HB * 16; h += 128) {
    float m = p.one > 0.f ? 0.f : -INFINITY, l = p.one;
    if (h < H && sp.ctx > 0)
      for (int s = 0; s < p.splits; ++s) {
        const float2 o = p.ml[((size_t)b * p.splits + s) * H + h];
        const float n = fmaxf(m, o.x);
        if (n > -INFINITY) l = l * tk_ex2(m - n) + o.y * tk_ex2(o.x - n);
        m = n;
      }
    s_z[h] = l > 0.f ? m + log2f(l) : 0.f;
  }
  for (int i = tid; i < HB * 16 * 8; i += 128) reinterpret_cast<uint4*>(sP)[i] = make_uint4(0, 0, 0, 0);       // rows past H stay zero
  uint32_t tf[HB][4];
#pragma unroll
  for (int j = 0; j < HB; ++j) talk_frag(p.talk, H, g * per, per, 16 * j, lane, tf[j]);
  float o[DV / 8][4];
#pragma unroll
  for (int n = 0; n < DV / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  const uint32_t ap = smem_u32(sP);
  __syncthreads();
  for (int page = sp.page; page < sp.end; ++page) {
    if (page + 1 < sp.end) fetch(page + 1);
    tk_commit();
    for (int i = tid; i < H * 16; i += 128) {              // four keys at a time
      const int h = i >> 4, c = (i & 15) * 4;
      const float4 s = *reinterpret_cast<const float4*>(p.scores + ((size_t)b * H + h) * p.band * TK_PAGE + page * TK_PAGE + c);
      const float z = s_z[h];
      *reinterpret_cast<uint2*>(sP + ms_off(h, c >> 3, 8) + (c & 7) * 2) = make_uint2(pack_half2(tk_ex2(s.x - z), tk_ex2(s.y - z)), pack_half2(tk_ex2(s.z - z), tk_ex2(s.w - z)));
    }
    tk_wait<1>();
    __syncthreads();
    // mixed weights of the warp's 16 keys, then their product with the values
    float m[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int j = 0; j < HB; ++j) {
      uint32_t b0, b1, b2, b3;
      ms_ldsm4t(ap + ms_off(16 * j + (lane & 7) + (((lane >> 3) & 1) << 3), 2 * warp + (lane >> 4), 8), b0, b1, b2, b3);
      mma_f16(m[0], tf[j], b0, b1);
      mma_f16(m[1], tf[j], b2, b3);
    }
    const uint32_t a[4] = {pack_bf16x2(m[0][0], m[0][1]), pack_bf16x2(m[0][2], m[0][3]), pack_bf16x2(m[1][0], m[1][1]), pack_bf16x2(m[1][2], m[1][3])};
    const uint32_t av = smem_u32(sV + (page & 1) * VB);
#pragma unroll
    for (int np = 0; np < DV / 16; ++np) {
      uint32_t b0, b1, b2, b3;
      ms_ldsm4t(av + ms_off(16 * warp + (((lane >> 3) & 1) << 3) + (lane & 7), 2 * np + (lane >> 4), VCH), b0, b1, b2, b3);
      ms_mma(o[2 * np], a, b0, b1);
      ms_mma(o[2 * np + 1], a, b2, b3);
    }
    __syncthreads();
  }
  tk_wait<0>();
  float* so = reinterpret_cast<float*>(sV);
#pragma unroll
  for (int n = 0; n < DV / 8; ++n)
#pragma unroll
    for (int e = 0; e < 2; ++e) *reinterpret_cast<float2*>(so + (warp * 16 + gq + 8 * e) * DV + 8 * n + 2 * tq) = make_float2(o[n][2 * e], o[n][2 * e + 1]);
  __syncthreads();
  for (int i = tid; i < per * p.dv; i += 128) {
    const int r = i / p.dv, c = i - r * p.dv;
    const float v = (so[r * DV + c] + so[(16 + r) * DV + c]) + (so[(32 + r) * DV + c] + so[(48 + r) * DV + c]);
    if (p.splits == 1) p.out[(size_t)b * p.ldo + (size_t)(g * per + r) * p.dv + c] = __float2bfloat16(v);
    else p.part[(((size_t)b * p.splits + split) * H + g * per + r) * p.dv + c] = v;
  }
}

// grid (blocks of 256 outputs, sequences): the splits' sums
__global__ void __launch_bounds__(256)
talk_merge_kernel(const TalkDecodeArgs p) {
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x * 256 + threadIdx.x, n = p.H * p.dv, b = blockIdx.y;
  if (i >= n) return;
  float v = 0.f;
  for (int s = 0; s < p.splits; ++s) v += p.part[((size_t)b * p.splits + s) * n + i];
  p.out[(size_t)b * p.ldo + i] = __float2bfloat16(v);
}

template <int KP, int HB, int NB>
static int talk_weights_launch(const TalkArgs& p, int batch, cudaStream_t s) {
  const int smem = p.H * 16 * KP * 2 + p.G * TW_KEYS * KP * 2 + HB * 16 * 1024 + p.H * 16 * 4 + 128;
  if (smem > 227 * 1024) return FF_HOST_TOO_LARGE;
  if (int r = opt_in_smem(talk_weights_kernel<KP, HB, NB>, smem)) return r;
  return launch_pdl(talk_weights_kernel<KP, HB, NB>, dim3(4 * p.tiles, p.parts, batch), dim3(256), smem, s, 0, p);
}
template <int KP, int HB>
static int talk_weights_batch(const TalkArgs& p, int batch, cudaStream_t s) {
  const int per = p.H / p.G;
  if (per >= 4 && p.G * ((per + 3) / 4) >= 8) return talk_weights_launch<KP, HB, 4>(p, batch, s);
  if (per >= 2 && p.G * ((per + 1) / 2) >= 8) return talk_weights_launch<KP, HB, 2>(p, batch, s);
  return talk_weights_launch<KP, HB, 1>(p, batch, s);
}
template <int KP>
static int talk_weights_heads(const TalkArgs& p, int batch, cudaStream_t s) {
  if (p.H <= 16) return talk_weights_batch<KP, 1>(p, batch, s);
  if (p.H <= 32) return talk_weights_batch<KP, 2>(p, batch, s);
  return FF_HOST_TOO_LARGE;
}
template <int DV, int NH>
static int talk_values_launch(const TalkArgs& p, int batch, cudaStream_t s) {
  const int per = p.H / p.G, smem = 2 * (NH * 64 * 128 + TK_PAGE * DV * 2) + 128;
  if (int r = opt_in_smem(talk_values_kernel<DV, NH>, smem)) return r;
  return launch_pdl(talk_values_kernel<DV, NH>, dim3(p.tiles, p.G * ((per + NH - 1) / NH), batch), dim3(64 * NH), smem, s, 0, p);
}
template <int DV>
static int talk_values_heads(const TalkArgs& p, int batch, cudaStream_t s) {
  const int per = p.H / p.G;
  if (per >= 3) return talk_values_launch<DV, 4>(p, batch, s);
  if (per == 2) return talk_values_launch<DV, 2>(p, batch, s);
  return talk_values_launch<DV, 1>(p, batch, s);
}

}  // namespace ff
using namespace ff;

// Mixed weights and value product of prompts. z [rows, H]: base-2 logarithm of every row's and head's soft-max denominator; scratch BF16
// [batch, tiles_per_round, H, 64, band * 64], band: the pages the 64 rows of a tile see at most; parts: CTAs that share a tile's keys; caches [num_blocks, G, 64, dk / dv].
// dk, dv multiples of 16 up to 128, H up to 32.
FF_EXPORT int ff_talk_prefill(const void* q, const void* kcache, const void* vcache, const int* block_table, const int* q_start, const int* q_lens,
                              const int* ctx_lens, const float* talk, const float* z, void* out, void* scratch, int batch, int max_q_len, int H, int G,
                              int dk, int dv, int ldq, int ldo, int max_blocks, int num_blocks, int window, int band, int tiles_per_round, int parts, float scale,
                              int* status, cudaStream_t s) {
  if (batch <= 0 || batch > 65535 || max_q_len <= 0 || H <= 0 || G <= 0 || H % G || window < 1 || band < 1 || tiles_per_round < 1 || parts < 1 || parts > 64 || scratch == nullptr) return FF_HOST_BAD_SHAPE;
  if (dk < 16 || dk > 128 || dk % 16 || dv < 16 || dv > 128 || dv % 16) return FF_HOST_BAD_SHAPE;
  if (ldq % 8 || ldo % 2 || (reinterpret_cast<uintptr_t>(q) & 15) || (reinterpret_cast<uintptr_t>(scratch) & 15) || (reinterpret_cast<uintptr_t>(out) & 3)) return FF_HOST_BAD_ALIGN;
  const int tiles = (max_q_len + 63) / 64;
  for (int t0 = 0; t0 < tiles; t0 += tiles_per_round) {
    const TalkArgs p = {(const __nv_bfloat16*)q, (const __nv_bfloat16*)kcache, (const __nv_bfloat16*)vcache, block_table, q_start, q_lens, ctx_lens, talk, z,
                        (__nv_bfloat16*)out, (__nv_bfloat16*)scratch, H, G, dk, dv, ldq, ldo, max_blocks, num_blocks, window, band, t0,
                        tiles - t0 < tiles_per_round ? tiles - t0 : tiles_per_round, parts, scale * TK_LOG2E, status};
    if (int r = dk <= 64 ? talk_weights_heads<64>(p, batch, s) : talk_weights_heads<128>(p, batch, s)) return r;
    if (int r = dv <= 64 ? talk_values_heads<64>(p, batch, s) : talk_values_heads<128>(p, batch, s)) return r;
  }
  return launch_result();
}

// One row per sequence. scores FP32 [batch, H, band * 64], ml float2 [batch, splits, H], part FP32 [batch, splits, H, dv] (splits > 1); one: the
// extra term of the denominator (0 or 1). dk, dv multiples of 16 up to 128, H up to 64, H / G up to 16.
FF_EXPORT int ff_talk_decode(const void* q, const void* kcache, const void* vcache, const int* block_table, const int* ctx_lens, const float* talk,
                             void* out, float* scores, float* ml, float* part, int batch, int H, int G, int dk, int dv, int ldq, int ldo, int max_blocks,
                             int num_blocks, int window, int band, int splits, float scale, float one, int* status, cudaStream_t s) {
  if (batch <= 0 || batch > 65535 || H <= 0 || G <= 0 || H % G || window < 1 || band < 1 || splits < 1 || !(one >= 0.f)) return FF_HOST_BAD_SHAPE;
  if (dk < 16 || dk > 128 || dk % 16 || dv < 16 || dv > 128 || dv % 16 || (splits > 1 && part == nullptr)) return FF_HOST_BAD_SHAPE;
  if (H > 64 || H / G > 16) return FF_HOST_TOO_LARGE;
  if (ldq % 8 || (reinterpret_cast<uintptr_t>(q) & 15)) return FF_HOST_BAD_ALIGN;
  const TalkDecodeArgs p = {(const __nv_bfloat16*)q, (const __nv_bfloat16*)kcache, (const __nv_bfloat16*)vcache, block_table, ctx_lens, talk,
                            (__nv_bfloat16*)out, scores, (float2*)ml, part, H, G, dk, dv, ldq, ldo, max_blocks, num_blocks, window, band, splits,
                            scale * TK_LOG2E, one, status};
  const dim3 grid(splits, G, batch);
  auto go = [&](auto kern, int smem) -> int {
    if (int r = opt_in_smem(kern, smem)) return r;
    return launch_pdl(kern, grid, dim3(128), smem, s, 0, p);
  };
  if (int r = dk <= 64 ? go(talk_scores_kernel<64>, 2 * TK_PAGE * 64 * 2 + 128) : go(talk_scores_kernel<128>, 2 * TK_PAGE * 128 * 2 + 128)) return r;
  const int vb = 2 * TK_PAGE * (dv <= 64 ? 64 : 128) * 2 + 128;        // the sums take as much: 4 * 16 rows of FP32
  int r;
  if (dv <= 64) r = H <= 16 ? go(talk_decode_kernel<64, 1>, vb) : H <= 32 ? go(talk_decode_kernel<64, 2>, vb) : go(talk_decode_kernel<64, 4>, vb);
  else r = H <= 16 ? go(talk_decode_kernel<128, 1>, vb) : H <= 32 ? go(talk_decode_kernel<128, 2>, vb) : go(talk_decode_kernel<128, 4>, vb);
  if (r) return r;
  if (splits > 1)
    if (int r2 = launch_pdl(talk_merge_kernel, dim3((H * dv + 255) / 256, batch), dim3(256), 0, s, 0, p)) return r2;
  return launch_result();
}
