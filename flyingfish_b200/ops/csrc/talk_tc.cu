// Windowed attention whose heads' weights are mixed before they meet the values (talk_simt.cu) on tensor cores: BF16, heads of up to 128
// elements, paged cache with 64-token pages.
//   w_g(i, j) = 2^(s_g(i, j) - z_g(i)),  z_g(i) the logarithm of the soft-max's denominator      M_h = sum_g talk[h, g] w_g      o_h = M_h v
// The mixed weights of a head need the normalised weights of every head, so no head can run its soft-max and its value product in one
// pass. Prompts take three, over tiles of 128 query rows:
//   1. talk_weights : scores on tcgen05 as in attention_tc.cu, 64 keys at a time; 2^(s - m) in FP16 goes to scratch by TMA, m being the
//                     maximum a thread has seen so far (two threads share a row, every other page each), and with it m of every 32
//                     keys and z at the end;
//   2. talk_mix     : a warp takes a query row, 64 keys of all heads at a time: the weights times 2^(m - z), then their product with the
//                     mixing matrix (mma.sync, heads as its inner dimension); mixed weights in BF16 replace the others in scratch;
//   3. talk_values  : scratch times values on tcgen05, two heads that share a value head per CTA.
// They go over a prompt in rounds that bound the scratch. Decoded tokens take two and a merge:
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

constexpr int TK_ROWS = 128;                 // query rows of a tile

struct TalkArgs {
  const int* block_table; const int* q_start; const int* q_lens; const int* ctx_lens;
  const float* talk;
  __nv_bfloat16* out;
  // a slot is one of the tiles worked on together: weights [slot, H, 128, band * 64], m [slot, H, band, 2 halves, 128], z [slot, H, 128]
  __nv_bfloat16* weights; float* m; float* z;
  int H, G, dk, dv, ldo, max_blocks, num_blocks, window, band;         // band: pages a tile's rows see at most
  int tile0, tiles;                          // the tiles worked on together
  float scale_log2, one;
  int* status;
};

// rows, positions and pages of a tile
struct TalkTile {
  int real, first, lo_page, pages;           // first: position of row 0
  __device__ TalkTile(const TalkArgs& p, int b, int tile) {
    const int qlen = p.q_lens[b], past = p.ctx_lens[b] - qlen, r0 = tile * TK_ROWS;
    real = min(TK_ROWS, qlen - r0);
    first = past + r0;
    lo_page = max(0, first - p.window + 1) / TK_PAGE;
    pages = min(p.band, (first + max(real, 1) - 1) / TK_PAGE - lo_page + 1);
  }
};
__device__ __forceinline__ int talk_page(const TalkArgs& p, int b, int page, bool& bad) {
  const int blk = p.block_table[(size_t)b * p.max_blocks + page];
  if (blk >= 0 && blk < p.num_blocks) return blk;
  bad = true;
  return 0;
}

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
// talk_weights: as many CTAs as fit, each takes every so many-th (sequence, tile, head). 320 threads: TMA warp, MMA warp, and two times
// four warps whose threads own a row of the even or of the odd pages. Shared memory: Q (two blocks of 64 columns), two K tiles, a staging
// tile of 32 rows and 64 keys per such warp. Tensor memory: four score tiles of 64 columns.
// ---------------------------------------------------------------------------------------
constexpr int TW_Q = TK_ROWS * 128 * 2, TW_K = TK_PAGE * 128 * 2, TW_P = 32 * TK_PAGE * 2;
constexpr int TW_SMEM = TW_Q + 2 * TW_K + 8 * TW_P + 1024;

struct alignas(8) TalkWeightBars {
  uint64_t q_full, q_empty, k_full[2], k_empty[2], s_full[4], s_empty[4];
  uint32_t tmem_base;
  int abort_flag;
  float m[2][TK_ROWS], l[2][TK_ROWS];        // of the odd pages; two, so that a head's do not meet the next one's
};

// (sequence, tile, head) number i
struct TalkItem {
  int b, tile, h;
  __device__ TalkItem(const TalkArgs& p, int i) { h = i % p.H; i /= p.H; tile = i % p.tiles; b = i / p.tiles; }
};

__global__ void __launch_bounds__(320, 2)
talk_weights_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmP,
                    const TalkArgs p, int items) {
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  extern __shared__ uint8_t tk_raw[];
  __shared__ TalkWeightBars bars;
  uint8_t* sQ = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tk_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sK = sQ + TW_Q;
  uint8_t* sP = sK + 2 * TW_K;
  const bool hi = p.dk > 64;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmP);
    mbar_init(&bars.q_full, 1); mbar_init(&bars.q_empty, 1);
    for (int i = 0; i < 2; ++i) { mbar_init(&bars.k_full[i], 1); mbar_init(&bars.k_empty[i], 1); }
    for (int i = 0; i < 4; ++i) { mbar_init(&bars.s_full[i], 1); mbar_init(&bars.s_empty[i], 4); }
    bars.abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(&bars.tmem_base, 256); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = bars.tmem_base;
  volatile int* abort_flag = &bars.abort_flag;
  int c = 0, n = 0;                                          // pages and items so far
  if (warp == 0) {
    if (lane == 0) {
      bool ok = true;
      for (int i = blockIdx.x; i < items && ok; i += gridDim.x) {
        const TalkItem it(p, i);
        const TalkTile tl(p, it.b, p.tile0 + it.tile);
        if (tl.real <= 0) continue;
        const int row = p.q_start[it.b] + (p.tile0 + it.tile) * TK_ROWS;
        if (!mbar_wait(&bars.q_empty, (n & 1) ^ 1, abort_flag, p.status, KID_ATTN_PREFILL, 40)) break;
        mbar_expect_tx(&bars.q_full, hi ? TW_Q : TW_Q / 2);
        tma_load_2d(sQ, &tmQ, &bars.q_full, it.h * p.dk, row);
        if (hi) tma_load_2d(sQ + TW_Q / 2, &tmQ, &bars.q_full, it.h * p.dk + 64, row);
        bool bad = false;
        for (int j = 0; j < tl.pages; ++j, ++c) {
          const int st = c & 1;
          const int krow = (talk_page(p, it.b, tl.lo_page + j, bad) * p.G + it.h / (p.H / p.G)) * TK_PAGE;
          ok = mbar_wait(&bars.k_empty[st], ((c >> 1) & 1) ^ 1, abort_flag, p.status, KID_ATTN_PREFILL, 41);
          if (!ok) break;
          mbar_expect_tx(&bars.k_full[st], hi ? TW_K : TW_K / 2);
          tma_load_2d(sK + st * TW_K, &tmK, &bars.k_full[st], 0, krow);
          if (hi) tma_load_2d(sK + st * TW_K + TW_K / 2, &tmK, &bars.k_full[st], 64, krow);
        }
        if (bad) set_status(p.status, KID_ATTN_PREFILL, FF_ERR_BOUNDS, it.b, p.tile0 + it.tile);
        ++n;
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = umma_idesc(1, 1, 0, 0, TK_ROWS, TK_PAGE), q_addr = smem_u32(sQ);
      const int ksteps = p.dk >> 4;
      bool ok = true;
      for (int i = blockIdx.x; i < items && ok; i += gridDim.x) {
        const TalkItem it(p, i);
        const TalkTile tl(p, it.b, p.tile0 + it.tile);
        if (tl.real <= 0) continue;
        ok = mbar_wait(&bars.q_full, n & 1, abort_flag, p.status, KID_ATTN_PREFILL, 42);
        for (int j = 0; j < tl.pages && ok; ++j, ++c) {
          const int st = c & 1, sb = c & 3;
          ok = mbar_wait(&bars.k_full[st], (c >> 1) & 1, abort_flag, p.status, KID_ATTN_PREFILL, 43) &&
               mbar_wait(&bars.s_empty[sb], ((c >> 2) & 1) ^ 1, abort_flag, p.status, KID_ATTN_PREFILL, 44);
          if (!ok) break;
          tc_fence_after();
          const uint32_t k_addr = smem_u32(sK + st * TW_K);
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            if (k >= ksteps) break;
            umma_f16(tmem_s + sb * TK_PAGE, umma_desc_sw128(q_addr + (k >> 2) * (TW_Q / 2) + (k & 3) * 32, 16, 1024),
                     umma_desc_sw128(k_addr + (k >> 2) * (TW_K / 2) + (k & 3) * 32, 16, 1024), idesc, k != 0);
          }
          umma_commit(&bars.s_full[sb]);
          umma_commit(&bars.k_empty[st]);
        }
        if (ok) umma_commit(&bars.q_empty);
        ++n;
      }
    }
  } else {
    const int q = warp & 3, odd = (warp - 2) >> 2, row = q * 32 + lane;
    uint8_t* stg = sP + (q * 2 + odd) * TW_P;
    const uint64_t scale2 = f2_pack(p.scale_log2, p.scale_log2);
    bool ok = true;
    for (int i = blockIdx.x; i < items; i += gridDim.x) {
      const TalkItem it(p, i);
      const TalkTile tl(p, it.b, p.tile0 + it.tile);
      if (tl.real <= 0) continue;
      const size_t slot_head = ((size_t)it.b * p.tiles + it.tile) * p.H + it.h;
      const int pos = tl.first + row;
      const bool live = row < tl.real;
      const int last = live ? pos : -1, from = live ? max(0, pos - p.window + 1) : 0;
      const int all_lo = max(0, tl.first + tl.real - p.window), all_hi = tl.real == TK_ROWS ? tl.first : -1;     // keys every row sees
      float m = -INFINITY, l = 0.f;
      for (int j = odd; j < tl.pages && ok; j += 2) {
        const int sb = (c + j) & 3;
        if (!mbar_wait(&bars.s_full[sb], ((c + j) >> 2) & 1, abort_flag, p.status, KID_ATTN_PREFILL, 45)) ok = false;
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
#pragma unroll 1
        for (int half = 0; half < 2; ++half) {
          float sv[32];
          {
            uint32_t r[32];
            tmem_ld_x32(tmem_s + (uint32_t(q * 32) << 16) + sb * TK_PAGE + 32 * half, r);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 32; ++e) sv[e] = __uint_as_float(r[e]);
          }
          if (half == 1) {
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&bars.s_empty[sb]);
          }
          const int k0 = (tl.lo_page + j) * TK_PAGE + 32 * half;
          float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
          if (!(k0 >= all_lo && k0 + 31 <= all_hi)) {
#pragma unroll
            for (int e = 0; e < 32; ++e) sv[e] = k0 + e >= from && k0 + e <= last ? sv[e] : -INFINITY;
          }
#pragma unroll
          for (int e = 0; e < 32; ++e) mx4[e & 3] = fmaxf(mx4[e & 3], sv[e]);
          const float mn = fmaxf(m, fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2), mr = mn == -INFINITY ? 0.f : mn;
          l *= m == -INFINITY ? 0.f : tk_ex2(m - mr);
          m = mn;
          p.m[((slot_head * p.band + j) * 2 + half) * TK_ROWS + row] = m;
          if (half == 0) {
            if (lane == 0) tma_store_wait_read<0>();         // the staging tile's previous contents have left
            __syncwarp();
          }
          const uint64_t neg = f2_pack(-mr, -mr);
          uint64_t ls[2] = {0ull, 0ull};
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            uint32_t w[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              float x, y;
              f2_unpack(f2_fma(f2_pack(sv[8 * e + 2 * k], sv[8 * e + 2 * k + 1]), scale2, neg), x, y);
              x = tk_ex2(x);
              y = tk_ex2(y);
              ls[k & 1] = f2_add(ls[k & 1], f2_pack(x, y));
              w[k] = pack_half2(x, y);
            }
            *reinterpret_cast<uint4*>(stg + lane * 128 + (((4 * half + e) ^ (lane & 7)) << 4)) = make_uint4(w[0], w[1], w[2], w[3]);
          }
          float la, lb;
          f2_unpack(f2_add(ls[0], ls[1]), la, lb);
          l += la + lb;
        }
        fence_proxy_async_smem();
        __syncwarp();
        if (lane == 0) {
          tma_store_2d(&tmP, stg, j * TK_PAGE, (int)(slot_head * TK_ROWS) + q * 32);
          tma_store_commit();
        }
      }
      if (odd) { bars.m[n & 1][row] = m; bars.l[n & 1][row] = l; }
      asm volatile("bar.sync 1, 256;" ::: "memory");
      if (!odd) {
        const float om = bars.m[n & 1][row], mx = fmaxf(fmaxf(m, om), p.one > 0.f ? 0.f : -INFINITY);
        p.z[slot_head * TK_ROWS + row] = mx == -INFINITY ? 0.f : mx + log2f(l * tk_ex2(m - mx) + bars.l[n & 1][row] * tk_ex2(om - mx) + (p.one > 0.f ? p.one * tk_ex2(-mx) : 0.f));
      }
      c += tl.pages;
      ++n;
    }
    if (lane == 0) tma_store_wait<0>();
  }
  tc_fence_before();
  __syncthreads();
  if (bars.abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) { __nanosleep(1000); }
  }
  if (warp == 1) { __syncwarp(); tc_fence_after(); tmem_dealloc(tmem_s, 256); }
}

// ---------------------------------------------------------------------------------------
// talk_mix: grid (16 * tiles, parts, sequences), 256 threads: eight neighbouring rows, a warp each, 64 keys of all heads at a time by TMA
// (one box of H rows of 128 bytes), three tiles per warp: two on their way in and one being worked on, which then is on its way out. HB: blocks of 16
// heads.
// ---------------------------------------------------------------------------------------
constexpr int TM_STAGES = 3;

__device__ __forceinline__ void stmatrix4(uint32_t a, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.shared.b16 [%0], {%1,%2,%3,%4};" ::"r"(a), "r"(r0), "r"(r1), "r"(r2), "r"(r3) : "memory");
}
__device__ __forceinline__ void talk_load_row(uint32_t dst, const CUtensorMap* m, uint64_t* bar, int key, int row, int slot) {
  asm volatile("cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6}], [%2];"
               ::"r"(dst), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(key), "r"(row), "r"(0), "r"(slot) : "memory");
}
__device__ __forceinline__ void talk_store_row(const CUtensorMap* m, uint32_t src, int key, int row, int slot) {
  asm volatile("cp.async.bulk.tensor.4d.global.shared::cta.bulk_group [%0, {%2, %3, %4, %5}], [%1];"
               ::"l"(reinterpret_cast<uint64_t>(m)), "r"(src), "r"(key), "r"(row), "r"(0), "r"(slot) : "memory");
}

template <int HB>
__global__ void __launch_bounds__(256, 2)
talk_mix_kernel(const __grid_constant__ CUtensorMap tmM, const TalkArgs p) {
  extern __shared__ __align__(128) uint8_t tk_raw[];
  constexpr int TB = HB * 16 * 128;                        // [heads][64 keys], 128-byte swizzle
  __shared__ uint64_t s_full[8][TM_STAGES];
  pdl_wait();
  const int b = blockIdx.z, slot = b * p.tiles + (blockIdx.x >> 4), row0 = (blockIdx.x & 15) * 8, H = p.H;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, tq = lane & 3;
  const TalkTile tl(p, b, p.tile0 + (blockIdx.x >> 4));
  const int rows = min(8, tl.real - row0);
  if (rows <= 0) return;
  // steps that some row sees, and this CTA's share of them
  const int pos = tl.first + row0, v0 = max(0, pos - p.window + 1) / TK_PAGE - tl.lo_page, v1 = min(tl.pages, (pos + rows - 1) / TK_PAGE - tl.lo_page + 1);
  const int j0 = v0 + (v1 - v0) * (int)blockIdx.y / (int)gridDim.y, j1 = v0 + (v1 - v0) * ((int)blockIdx.y + 1) / (int)gridDim.y, n = j1 - j0;
  if (n <= 0) return;
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tk_raw) + 1023) & ~uintptr_t(1023));
  __half* s_f = reinterpret_cast<__half*>(base + 8 * TM_STAGES * TB);  // [step][row][half][heads]
  const uint32_t buf = smem_u32(base) + warp * TM_STAGES * TB;
  uint64_t* full = s_full[warp];
  if (lane == 0) {
    for (int i = 0; i < TM_STAGES; ++i) mbar_init(&full[i], 1);
    mbar_fence_init();
  }
  for (int i = H * 8 + lane; i < HB * 16 * 8; i += 32)     // heads past H
    for (int st = 0; st < TM_STAGES; ++st)
      asm volatile("st.shared.v4.b32 [%0], {%1,%1,%1,%1};" ::"r"(buf + st * TB + ms_off(i >> 3, i & 7, 8)), "r"(0) : "memory");
  __syncwarp();
  const bool live = warp < rows;
  if (live && lane == 0)
    for (int k = 0; k < min(n, 2); ++k) {
      mbar_expect_tx(&full[k], H * 128);
      talk_load_row(buf + k * TB, &tmM, &full[k], (j0 + k) * TK_PAGE, row0 + warp, slot);
    }
  // the factors 2^(m - z) of all steps: a thread takes a row and heads tid / 8, + 32
  for (int h = tid >> 3; h < HB * 16; h += 32) {
    const int r = tid & 7;
    const size_t sh = (size_t)slot * H + min(h, H - 1);
    const float z = p.z[sh * TK_ROWS + row0 + r];
    const float* mp = p.m + (sh * p.band + j0) * 2 * TK_ROWS + row0 + r;
    for (int k0 = 0; k0 < 2 * n; k0 += 8) {                // eight loads on their way together
      float m[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) m[e] = mp[(size_t)min(k0 + e, 2 * n - 1) * TK_ROWS];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int k = k0 + e;
        if (k < 2 * n) s_f[((k >> 1) * 16 + 2 * r + (k & 1)) * HB * 16 + h] = __float2half(h < H ? tk_ex2(m[e] - z) : 0.f);
      }
    }
  }
  uint32_t tf[HB][HB][4];
#pragma unroll
  for (int i = 0; i < HB; ++i)
#pragma unroll
    for (int k = 0; k < HB; ++k) talk_frag(p.talk, H, 16 * i, 16, 16 * k, lane, tf[i][k]);
  __syncthreads();
  if (!live) return;
  const int r16 = (lane & 7) + (((lane >> 3) & 1) << 3);
  int st = 0; uint32_t ph = 0;
  for (int k = 0; k < n; ++k) {
    if (!mbar_wait(&full[st], ph, nullptr, p.status, KID_ATTN_PREFILL, 61)) break;
    __syncwarp();
    const uint32_t d = buf + st * TB;
    const uint32_t* fr = reinterpret_cast<const uint32_t*>(s_f + (k * 16 + 2 * warp) * HB * 16);
#pragma unroll
    for (int c = 0; c < 8; c += 2) {                       // 16 keys of all heads
      const uint32_t at = d + r16 * 128 + (((c + (lane >> 4)) ^ (lane & 7)) << 4);
      uint32_t bf[HB][4];
#pragma unroll
      for (int i = 0; i < HB; ++i) {
        ms_ldsm4t(at + i * 2048, bf[i][0], bf[i][1], bf[i][2], bf[i][3]);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const uint32_t f = fr[((c >> 2) * HB * 16 + 16 * i + 8 * e) / 2 + tq];
          const __half2 x = __hmul2(*reinterpret_cast<const __half2*>(&bf[i][e]), *reinterpret_cast<const __half2*>(&f));
          const __half2 y = __hmul2(*reinterpret_cast<const __half2*>(&bf[i][2 + e]), *reinterpret_cast<const __half2*>(&f));
          bf[i][e] = *reinterpret_cast<const uint32_t*>(&x);
          bf[i][2 + e] = *reinterpret_cast<const uint32_t*>(&y);
        }
      }
      float a[HB][2][4];
#pragma unroll
      for (int i = 0; i < HB; ++i) {
#pragma unroll
        for (int e = 0; e < 4; ++e) a[i][0][e] = a[i][1][e] = 0.f;
#pragma unroll
        for (int q = 0; q < HB; ++q) { mma_f16(a[i][0], tf[i][q], bf[q][0], bf[q][1]); mma_f16(a[i][1], tf[i][q], bf[q][2], bf[q][3]); }
      }
      __syncwarp();                                        // these keys are in registers: their place takes the result
#pragma unroll
      for (int i = 0; i < HB; ++i)
        stmatrix4(at + i * 2048, pack_bf16x2(a[i][0][0], a[i][0][1]), pack_bf16x2(a[i][0][2], a[i][0][3]), pack_bf16x2(a[i][1][0], a[i][1][1]),
                  pack_bf16x2(a[i][1][2], a[i][1][3]));
    }
    fence_proxy_async_smem();
    __syncwarp();
    if (lane == 0) {
      if (k + 2 < n) {
        const int free = st == 0 ? TM_STAGES - 1 : st - 1;
        tma_store_wait_read<0>();                          // the tile that left from there
        mbar_expect_tx(&full[free], H * 128);
        talk_load_row(buf + free * TB, &tmM, &full[free], (j0 + k + 2) * TK_PAGE, row0 + warp, slot);
      }
      talk_store_row(&tmM, d, (j0 + k) * TK_PAGE, row0 + warp, slot);
      tma_store_commit();
    }
    if (++st == TM_STAGES) { st = 0; ph ^= 1; }
  }
  if (lane == 0) tma_store_wait<0>();
}

// ---------------------------------------------------------------------------------------
// talk_values: grid (tiles, G * batches of NH heads, sequences), 192 threads: TMA warp, MMA warp, four warps that store the result. Two
// stages of NH weight tiles [128 rows, 64 keys] and a page of values.
// ---------------------------------------------------------------------------------------
constexpr int TV_W = TK_ROWS * TK_PAGE * 2, TV_V = TK_PAGE * 128 * 2, TV_STAGES = 2;
struct alignas(8) TalkValueBars {
  uint64_t full[TV_STAGES], empty[TV_STAGES], done;
  uint32_t tmem_base;
  int abort_flag;
};

template <int NH>
__global__ void __launch_bounds__(192, 2)
talk_values_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmV, const TalkArgs p) {
  pdl_wait();
  const int b = blockIdx.z, tile = p.tile0 + blockIdx.x, per = p.H / p.G, batches = (per + NH - 1) / NH, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = blockIdx.y / batches, h0 = g * per + (blockIdx.y % batches) * NH, heads = min(NH, (g + 1) * per - h0);
  const TalkTile tl(p, b, tile);
  if (tl.real <= 0) return;
  extern __shared__ uint8_t tk_raw[];
  __shared__ TalkValueBars bars;
  constexpr int STAGE = NH * TV_W + TV_V;
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tk_raw) + 1023) & ~uintptr_t(1023));
  const bool hi = p.dv > 64;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmW); tma_prefetch_desc(&tmV);
    for (int i = 0; i < TV_STAGES; ++i) { mbar_init(&bars.full[i], 1); mbar_init(&bars.empty[i], 1); }
    mbar_init(&bars.done, 1);
    bars.abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(&bars.tmem_base, NH * 128); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_o = bars.tmem_base;
  volatile int* abort_flag = &bars.abort_flag;
  if (warp == 0) {
    if (lane == 0) {
      const int wrow = (((int)b * p.tiles + (int)blockIdx.x) * p.H + h0) * TK_ROWS;
      bool bad = false;
      for (int j = 0; j < tl.pages; ++j) {
        const int st = j % TV_STAGES; const uint32_t ph = (j / TV_STAGES) & 1;
        const int vrow = (talk_page(p, b, tl.lo_page + j, bad) * p.G + g) * TK_PAGE;
        if (!mbar_wait(&bars.empty[st], ph ^ 1, abort_flag, p.status, KID_ATTN_PREFILL, 51)) break;
        uint8_t* at = sm + st * STAGE;
        mbar_expect_tx(&bars.full[st], heads * TV_W + (hi ? TV_V : TV_V / 2));
        for (int n = 0; n < heads; ++n) tma_load_2d(at + n * TV_W, &tmW, &bars.full[st], j * TK_PAGE, wrow + n * TK_ROWS);
        tma_load_2d(at + NH * TV_W, &tmV, &bars.full[st], 0, vrow);
        if (hi) tma_load_2d(at + NH * TV_W + TV_V / 2, &tmV, &bars.full[st], 64, vrow);
      }
      if (bad) set_status(p.status, KID_ATTN_PREFILL, FF_ERR_BOUNDS, b, tile);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = umma_idesc(1, 1, 0, 1, TK_ROWS, hi ? 128 : 64);
      bool ok = true;
      for (int j = 0; j < tl.pages && ok; ++j) {
        const int st = j % TV_STAGES; const uint32_t ph = (j / TV_STAGES) & 1;
        if (!mbar_wait(&bars.full[st], ph, abort_flag, p.status, KID_ATTN_PREFILL, 52)) { ok = false; break; }
        tc_fence_after();
        const uint32_t at = smem_u32(sm + st * STAGE), v_addr = at + NH * TV_W;
        for (int n = 0; n < heads; ++n)
#pragma unroll
          for (int k = 0; k < TK_PAGE / 16; ++k)
            umma_f16(tmem_o + n * 128, umma_desc_sw128(at + n * TV_W + k * 32, 16, 1024), umma_desc_sw128(v_addr + k * 2048, TV_V / 2, 1024), idesc, (j | k) != 0);
        umma_commit(&bars.empty[st]);
      }
      if (ok) umma_commit(&bars.done);
    }
  } else {
    const int q = warp & 3, row = q * 32 + lane;
    bool ok = mbar_wait(&bars.done, 0, abort_flag, p.status, KID_ATTN_PREFILL, 53);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tc_fence_after();
      for (int n = 0; n < heads; ++n) {
        __nv_bfloat16* dst = p.out + (size_t)(p.q_start[b] + tile * TK_ROWS + row) * p.ldo + (size_t)(h0 + n) * p.dv;
        for (int c = 0; c < p.dv; c += 16) {
          uint32_t r[16];
          tmem_ld_x16(tmem_o + (uint32_t(q * 32) << 16) + n * 128 + c, r);
          tmem_ld_wait();
          if (row < tl.real) {
            uint32_t o[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) o[i] = pack_bf16x2(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1]));
            reinterpret_cast<uint4*>(dst + c)[0] = make_uint4(o[0], o[1], o[2], o[3]);
            reinterpret_cast<uint4*>(dst + c)[1] = make_uint4(o[4], o[5], o[6], o[7]);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (bars.abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) { __nanosleep(1000); }
  }
  if (warp == 1) { __syncwarp(); tc_fence_after(); tmem_dealloc(tmem_o, NH * 128); }
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
    const int pages = ctx > 0 ? min(p.band, (ctx - 1) / TK_PAGE - lo_page + 1) : 0, each = (pages + p.splits - 1) / p.splits;
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

// weights as (key, row, head, slot), boxes of 64 keys of all heads
static int talk_row_map(CUtensorMap* out, void* base, uint64_t bandw, uint64_t heads, uint64_t slots) {
  EncodeTiledFn fn = encode_tiled_fn();
  if (!fn) return FF_HOST_NO_DRIVER;
  const cuuint64_t dims[4] = {bandw, TK_ROWS, heads, slots}, strides[3] = {bandw * 2, bandw * 2 * TK_ROWS, bandw * 2 * TK_ROWS * heads};
  const cuuint32_t box[4] = {TK_PAGE, 1, (cuuint32_t)heads, 1}, step[4] = {1, 1, 1, 1};
  const CUresult r = fn(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, base, dims, strides, box, step, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                        CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? FF_HOST_OK : FF_HOST_TMAP_FAIL;
}

template <int HB>
static int talk_mix_launch(const CUtensorMap& tmM, const TalkArgs& p, int batch, cudaStream_t s) {
  // CTAs that share a row's keys: enough for the device, and few enough steps each for the factors
  const int groups = batch * p.tiles * (TK_ROWS / 8), fit = 2 * sm_count(), most = HB == 1 ? 32 : 16;
  int parts = groups < fit ? fit / groups : 1;
  if (parts < (p.band + most - 1) / most) parts = (p.band + most - 1) / most;
  const int steps = (p.band + parts - 1) / parts, smem = 8 * TM_STAGES * HB * 16 * 128 + steps * 16 * HB * 16 * 2 + 1024;
  if (parts > 65535) return FF_HOST_TOO_LARGE;
  if (int r = opt_in_smem(talk_mix_kernel<HB>, smem)) return r;
  return launch_pdl(talk_mix_kernel<HB>, dim3(16 * p.tiles, parts, batch), dim3(256), smem, s, 0, tmM, p);
}
template <int NH>
static int talk_values_launch(const CUtensorMap& tmW, const CUtensorMap& tmV, const TalkArgs& p, int batch, cudaStream_t s) {
  const int per = p.H / p.G, smem = TV_STAGES * (NH * TV_W + TV_V) + 1024;
  if (int r = opt_in_smem(talk_values_kernel<NH>, smem)) return r;
  return launch_pdl(talk_values_kernel<NH>, dim3(p.tiles, p.G * ((per + NH - 1) / NH), batch), dim3(192), smem, s, 0, tmW, tmV, p);
}

}  // namespace ff
using namespace ff;

// Prompts. q: packed rows [total_rows, ldq] with head h at column h * dk; caches [num_blocks, G, 64, dk / dv]; talk FP32 [H, H]; out rows of
// pitch ldo; scratch: batch * tiles_per_round slots of H * 128 * (34 band + 1) floats; the call takes the rounds
// first_round, first_round + round_step, ..; one: the extra term of the
// denominator (0 or 1). dk, dv multiples of 16 up to 128, H up to 32.
FF_EXPORT int ff_talk_prefill(const void* q, const void* kcache, const void* vcache, const int* block_table, const int* q_start, const int* q_lens,
                              const int* ctx_lens, const float* talk, void* out, float* scratch, int batch, int total_rows, int max_q_len, int H, int G,
                              int dk, int dv, int ldq, int ldo, int max_blocks, int num_blocks, int window, int band, int tiles_per_round, int first_round, int round_step,
                              float scale, float one, int* status, cudaStream_t s) {
  if (batch <= 0 || batch > 65535 || total_rows <= 0 || max_q_len <= 0 || H <= 0 || G <= 0 || H % G || window < 1 || band < 1 || tiles_per_round < 1 ||
      first_round < 0 || round_step < 1 || scratch == nullptr || !(scale > 0.f) || !(one >= 0.f)) return FF_HOST_BAD_SHAPE;
  if (dk < 16 || dk > 128 || dk % 16 || dv < 16 || dv > 128 || dv % 16 || ldq < H * dk || ldo < H * dv) return FF_HOST_BAD_SHAPE;
  const long long rows = (long long)batch * tiles_per_round * H * TK_ROWS;
  if (H > 32 || rows > (1ll << 30)) return FF_HOST_TOO_LARGE;
  if (ldq % 8 || ldo % 8 || (reinterpret_cast<uintptr_t>(scratch) & 15) || (reinterpret_cast<uintptr_t>(out) & 15)) return FF_HOST_BAD_ALIGN;
  constexpr auto BF = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;    // weights: two bytes either way
  const uint64_t bandw = (uint64_t)band * TK_PAGE, cache_rows = (uint64_t)num_blocks * G * TK_PAGE;
  CUtensorMap tmQ, tmK, tmV, tmP, tmW, tmM;
  if (int r = make_tmap_2d(&tmQ, q, BF, 2, (uint64_t)ldq, total_rows, (uint64_t)ldq * 2, 64, TK_ROWS)) return r;
  if (int r = make_tmap_2d(&tmK, kcache, BF, 2, dk, cache_rows, (uint64_t)dk * 2, 64, TK_PAGE)) return r;
  if (int r = make_tmap_2d(&tmV, vcache, BF, 2, dv, cache_rows, (uint64_t)dv * 2, 64, TK_PAGE)) return r;
  if (int r = make_tmap_2d(&tmP, scratch, BF, 2, bandw, rows, bandw * 2, 64, 32)) return r;
  if (int r = make_tmap_2d(&tmW, scratch, BF, 2, bandw, rows, bandw * 2, 64, TK_ROWS)) return r;
  if (int r = talk_row_map(&tmM, scratch, bandw, H, (uint64_t)batch * tiles_per_round)) return r;
  if (int r = opt_in_smem(talk_weights_kernel, TW_SMEM)) return r;
  float* m = scratch + rows * (long long)bandw / 2;
  const int tiles = (max_q_len + TK_ROWS - 1) / TK_ROWS;
  for (int t0 = first_round * tiles_per_round; t0 < tiles; t0 += round_step * tiles_per_round) {
    const TalkArgs p = {block_table, q_start, q_lens, ctx_lens, talk, (__nv_bfloat16*)out, (__nv_bfloat16*)scratch, m, m + 2 * rows * band, H, G, dk, dv, ldo,
                        max_blocks, num_blocks, window, band, t0, tiles - t0 < tiles_per_round ? tiles - t0 : tiles_per_round, scale * TK_LOG2E, one, status};
    const int items = batch * p.tiles * H, fit = 2 * sm_count();
    if (int r = launch_pdl(talk_weights_kernel, dim3(items < fit ? items : fit), dim3(320), TW_SMEM, s, 0, tmQ, tmK, tmP, p, items)) return r;
    if (int r = H <= 16 ? talk_mix_launch<1>(tmM, p, batch, s) : talk_mix_launch<2>(tmM, p, batch, s)) return r;
    if (int r = H / G >= 2 ? talk_values_launch<2>(tmW, tmV, p, batch, s) : talk_values_launch<1>(tmW, tmV, p, batch, s)) return r;
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
