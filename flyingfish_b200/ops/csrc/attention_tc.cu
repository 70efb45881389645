// Prefill attention on 5th-generation tensor cores: paged KV, heads of up to 128 elements, GQA, causal / sliding-window /
// block-local / bidirectional masks, a sliding window that keeps the first positions, soft-capped scores, optional output gate (per
// element or per head), chunked prefill (query rows are the last q_len positions of a context of ctx_len).
//
// One CTA per (sequence, query head, tile of 128 query rows). Both contractions run as tcgen05.mma with
// FP32 accumulators in tensor memory:
//
//   S = Q Kᵀ      A = Q tile  [128 rows x 128 d]   (K-major, two 64-column blocks, 128-byte swizzle, TMA)
//                 B = K tile  [128 keys x 128 d]   (K-major, two pages of the cache, TMA)
//                 D = S       TMEM, 128 lanes x 128 columns, double-buffered so that Q K(j+1)ᵀ runs while the
//                             softmax warps work on tile j
//   O += P V      A = P tile  [128 rows x 128 keys] BF16, written by the softmax warps into 128-byte-swizzled
//                             shared memory (K-major over keys)
//                 B = V tile  [128 keys x 128 d]    exactly as the cache stores it: d contiguous = MN-major
//                 D = O       TMEM, 128 lanes x 128 columns, lives across all KV tiles
//
// Warp roles: warp 0 = TMA producer (Q once, then K tiles through a ring of two and V tiles through a ring of three
// stages -- a K tile is released right after its Q Kᵀ, so the loads run two tiles ahead; block ids read from the
// block table), warp 1 = MMA issuer, warps 2-9 = softmax: two threads share query row t (TMEM lane t) and split its
// key columns in halves (two warps per lane quadrant, so each scheduler has two warps to interleave); a thread reads its S
// row with tcgen05.ld, applies the mask where a tile needs one, keeps the running maximum and sum in the base-2 domain
// (scale folded into the exponent's FMA, ex2.approx straight on the MUFU), and
// rescales O in TMEM only when the maximum has moved by more than 2^8 (the stale maximum stays exact: P and
// the sum use the same reference, the final division cancels it).
//
// Every wait is bounded; a time-out records FF_ERR_TIMEOUT and the CTA leaves through the abort flag, frees
// its tensor memory and returns. Replaces the mma.sync prefill kernel of attention_paged.cu (kept for
// comparison) and the reference's FlashAttention-2 adapter / Rust-PTX prefill kernels
// (third_party/flash-attention/adapter.cu:147-162, device/src/lib.rs:422-940).
#include "ptx.cuh"
#include "host_util.h"

namespace ff {

__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

constexpr int TC_HD = 128, TC_PAGE = 64, TC_BM = 128, TC_BN = 128;
constexpr int TC_KSTAGES = 3, TC_VSTAGES = 3;             // K is done with after Q Kᵀ, V only after P V: separate rings
constexpr int TC_Q_BYTES = TC_BM * TC_HD * 2;             // 32 KiB
constexpr int TC_KV_BYTES = TC_BN * TC_HD * 2;            // 32 KiB per operand per stage
constexpr int TC_SMEM = TC_Q_BYTES + (TC_KSTAGES + TC_VSTAGES) * TC_KV_BYTES + 1024;   // 225 KiB
constexpr float TC_RESCALE_THRESHOLD = 8.0f;              // log2 units
constexpr int TC_TWO_CTAS_DEFAULT = 1;
constexpr int TC2_SPLIT_DEFAULT = 1;

struct alignas(8) TcBars {
  uint64_t q_full;
  uint64_t k_full[TC_KSTAGES];
  uint64_t k_empty[TC_KSTAGES];
  uint64_t v_full[TC_VSTAGES];
  uint64_t v_empty[TC_VSTAGES];
  uint64_t s_full[2];
  uint64_t s_empty[2];
  uint64_t p_full;
  uint64_t p_empty;
  uint64_t o_done;
  uint32_t tmem_base;
  int abort_flag;
  float xmax[2][TC_BM];      // row maxima (and, at the end, row sums) exchanged between the two warps of a quadrant
};

__global__ void __launch_bounds__(320, 1)
attn_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                       const __grid_constant__ CUtensorMap tmV, const int* __restrict__ block_table,
                       const int* __restrict__ q_start, const int* __restrict__ q_lens,
                       const int* __restrict__ ctx_lens, __nv_bfloat16* __restrict__ out, int hq, int hkv, int ldo,
                       int max_blocks, int num_blocks, float scale_log2, int window, int causal, int* status,
                       const float* __restrict__ sinks) {
  const int b = blockIdx.z, h = blockIdx.y;
  const int qlen = q_lens[b];
  // later query tiles of a causal prefill see more keys: they are scheduled first so that the long CTAs do not form the tail
  const int r0 = (gridDim.x - 1 - blockIdx.x) * TC_BM;
  if (r0 >= qlen) return;
  extern __shared__ uint8_t smem_raw[];
  __shared__ TcBars bars;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sKr = smem + TC_Q_BYTES;                       // K ring, then V ring: 32 KiB tiles
  uint8_t* sVr = sKr + TC_KSTAGES * TC_KV_BYTES;
  const int ctx = ctx_lens[b], qs = q_start[b];
  const int kvh = h / (hq / hkv);
  const int past = ctx - qlen;
  const int real = min(TC_BM, qlen - r0);
  // key range of this tile
  const int last_key = causal ? past + r0 + real - 1 : ctx - 1;
  const int first_key = window > 0 ? max(0, past + r0 - window + 1) : 0;
  const int t0 = first_key / TC_BN, t1 = last_key / TC_BN + 1;
  const int ntiles = t1 - t0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
    mbar_init(&bars.q_full, 1);
    for (int i = 0; i < TC_KSTAGES; ++i) { mbar_init(&bars.k_full[i], 1); mbar_init(&bars.k_empty[i], 1); }
    for (int i = 0; i < TC_VSTAGES; ++i) { mbar_init(&bars.v_full[i], 1); mbar_init(&bars.v_empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&bars.s_full[i], 1); mbar_init(&bars.s_empty[i], 8); }
    mbar_init(&bars.p_full, 1); mbar_init(&bars.p_empty, 1); mbar_init(&bars.o_done, 1);
    bars.abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(&bars.tmem_base, 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = bars.tmem_base;
  const uint32_t tmem_o = tmem_base + 256;
  const uint32_t tmem_p = tmem_base + 384;       // P: 128 keys as 64 columns of packed BF16 pairs
  volatile int* abort_flag = &bars.abort_flag;

  if (warp == 0) {
    // ================================ TMA producer ================================
    if (lane == 0) {
      mbar_expect_tx(&bars.q_full, TC_Q_BYTES);
      // rows past the sequence's own belong to the next sequence of the packed batch (or are out of range and read
      // as zero): their lanes are computed and never stored
      tma_load_2d(sQ, &tmQ, &bars.q_full, h * TC_HD, qs + r0);
      tma_load_2d(sQ + TC_BM * 128, &tmQ, &bars.q_full, h * TC_HD + 64, qs + r0);
      bool ok = true, bad = false;
      const int nblk = (ctx + TC_PAGE - 1) / TC_PAGE;
      for (int j = 0; j < ntiles && ok; ++j) {
        const int ks = j % TC_KSTAGES, vs = j % TC_VSTAGES;
        int rows[2];
        for (int pg = 0; pg < 2; ++pg) {
          int page = (t0 + j) * 2 + pg;
          if (page >= nblk) page = nblk - 1;                 // past the context: any valid page, its keys are masked
          int blk = block_table[(size_t)b * max_blocks + page];
          if (blk < 0 || blk >= num_blocks) { bad = true; blk = 0; }
          rows[pg] = (blk * hkv + kvh) * TC_PAGE;
        }
        // layout of a tile: block d0 = [128 keys x 64 d] (16 KiB), then block d1; a page is 64 keys of each
        if (!mbar_wait(&bars.k_empty[ks], ((j / TC_KSTAGES) & 1) ^ 1, abort_flag, status, KID_ATTN_PREFILL, 1)) { ok = false; break; }
        mbar_expect_tx(&bars.k_full[ks], TC_KV_BYTES);
        uint8_t* sK = sKr + ks * TC_KV_BYTES;
        for (int pg = 0; pg < 2; ++pg) {
          tma_load_2d(sK + pg * 8192, &tmK, &bars.k_full[ks], 0, rows[pg]);
          tma_load_2d(sK + 16384 + pg * 8192, &tmK, &bars.k_full[ks], 64, rows[pg]);
        }
        if (!mbar_wait(&bars.v_empty[vs], ((j / TC_VSTAGES) & 1) ^ 1, abort_flag, status, KID_ATTN_PREFILL, 10)) { ok = false; break; }
        mbar_expect_tx(&bars.v_full[vs], TC_KV_BYTES);
        uint8_t* sV = sVr + vs * TC_KV_BYTES;
        for (int pg = 0; pg < 2; ++pg) {
          tma_load_2d(sV + pg * 8192, &tmV, &bars.v_full[vs], 0, rows[pg]);
          tma_load_2d(sV + 16384 + pg * 8192, &tmV, &bars.v_full[vs], 64, rows[pg]);
        }
      }
      if (bad) set_status(status, KID_ATTN_PREFILL, FF_ERR_BOUNDS, b, r0 / TC_BM);
    }
  } else if (warp == 1) {
    // ================================ MMA issuer ================================
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc(1, 1, 0, 0, TC_BM, TC_BN);      // Q (K-major) x K (K-major)
      const uint32_t idesc_o = umma_idesc(1, 1, 0, 1, TC_BM, TC_HD);      // P (K-major) x V (MN-major)
      const uint32_t q_addr = smem_u32(sQ);
      bool ok = mbar_wait(&bars.q_full, 0, abort_flag, status, KID_ATTN_PREFILL, 2);
      auto issue_s = [&](int j) -> bool {
        const int ks = j % TC_KSTAGES; const uint32_t ph = (j / TC_KSTAGES) & 1;
        const int sb = j & 1; const uint32_t sph = (j >> 1) & 1;
        if (!mbar_wait(&bars.k_full[ks], ph, abort_flag, status, KID_ATTN_PREFILL, 3)) return false;
        if (!mbar_wait(&bars.s_empty[sb], sph ^ 1, abort_flag, status, KID_ATTN_PREFILL, 4)) return false;
        tc_fence_after();
        const uint32_t k_addr = smem_u32(sKr + ks * TC_KV_BYTES);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const uint32_t off = (k >> 2) * 16384 + (k & 3) * 32;
          umma_f16(tmem_base + sb * TC_BN, umma_desc_sw128(q_addr + off, 16, 1024), umma_desc_sw128(k_addr + off, 16, 1024),
                   idesc_s, k != 0);
        }
        umma_commit(&bars.s_full[sb]);
        umma_commit(&bars.k_empty[ks]);            // the K tile is free as soon as this product has read it
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; j < ntiles && ok; ++j) {
        if (j + 1 < ntiles) { ok = issue_s(j + 1); if (!ok) break; }
        if (!mbar_wait(&bars.p_full, j & 1, abort_flag, status, KID_ATTN_PREFILL, 5)) { ok = false; break; }
        const int vs = j % TC_VSTAGES;
        if (!mbar_wait(&bars.v_full[vs], (j / TC_VSTAGES) & 1, abort_flag, status, KID_ATTN_PREFILL, 11)) { ok = false; break; }
        tc_fence_after();
        const uint32_t v_addr = smem_u32(sVr + vs * TC_KV_BYTES);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          // P: the 16 keys of k-step k are 8 columns of the P region of tensor memory; V: 16 key rows = 2 KiB
          const uint64_t db = umma_desc_sw128(v_addr + (k >> 2) * 8192 + (k & 3) * 2048, 16384, 1024);
          umma_f16_ts(tmem_o, tmem_p + k * 8, db, idesc_o, (j > 0) || (k != 0));
        }
        umma_commit(&bars.p_empty);
        umma_commit(&bars.v_empty[vs]);
      }
      if (ok) umma_commit(&bars.o_done);
    }
  } else {
    // ================================ softmax warps 2..9 ================================
    // Two warps per 32-lane quadrant of tensor memory (a warp may only touch the lanes of quadrant warp % 4): the pair
    // shares the rows of its quadrant and splits a tile's 128 key columns (and O's 128 columns, when it is rescaled)
    // in halves, so every scheduler has two warps to interleave. Row maxima cross the pair through shared memory.
    const int q = warp & 3;
    const int hf = (warp - 2) >> 2;               // which 64-column half this warp owns
    const int row = q * 32 + lane;                // query row of the tile = TMEM lane
    const int e = (warp - 2) * 32 + lane;
    const bool live = row < real;
    const int pos = past + r0 + row;              // absolute position of the row
    const int hi = live ? (causal ? pos : ctx - 1) : -1;
    const int lo = (live && window > 0) ? max(0, pos - window + 1) : 0;
    float m_ref = -INFINITY, l_sum = 0.f;
    bool ok = true;
    const uint32_t lane_base = (uint32_t(q * 32) << 16);
    // key range common to all live rows of the tile: [largest lower bound, smallest upper bound]
    const int tile_hi_min = causal ? past + r0 : ctx - 1;
    const int tile_lo_max = window > 0 ? max(0, past + r0 + real - window) : 0;
    constexpr int HB = TC_BN / 2;                 // columns per warp
    // A wait that gives up clears `ok` for the whole warp; the warp then skips the work of the remaining tiles but still
    // takes part in every barrier, so that no other warp is left waiting for it.
    for (int j = 0; j < ntiles; ++j) {
      const int sb = j & 1; const uint32_t sph = (j >> 1) & 1;
      if (ok && !mbar_wait(&bars.s_full[sb], sph, abort_flag, status, KID_ATTN_PREFILL, 6)) ok = false;
      ok = __all_sync(0xffffffffu, ok);
      float sv[HB];
      float mx = -INFINITY;
      if (ok) {
      tc_fence_after();
      {
        uint32_t r[HB];
#pragma unroll
        for (int c = 0; c < HB; c += 32) tmem_ld_x32(tmem_base + lane_base + sb * TC_BN + hf * HB + c, r + c);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < HB; ++i) sv[i] = __uint_as_float(r[i]);
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars.s_empty[sb]);
      const int k0 = (t0 + j) * TC_BN + hf * HB;
      // sv stays in raw score units: the scale is folded into the exponent's FMA below. A tile that lies inside the key
      // range of every live row of this query tile (most tiles of a long context) skips the mask altogether.
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      if ((t0 + j) * TC_BN >= tile_lo_max && (t0 + j) * TC_BN + TC_BN - 1 <= tile_hi_min) {
#pragma unroll
        for (int i = 0; i < HB; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], sv[i]);
      } else {
#pragma unroll
        for (int i = 0; i < HB; ++i) {
          const int key = k0 + i;
          const float t = (key >= lo && key <= hi) ? sv[i] : -INFINITY;
          sv[i] = t;
          mx4[i & 3] = fmaxf(mx4[i & 3], t);
        }
      }
      mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale_log2;   // scale > 0 commutes with the maximum
      }
      // the row's maximum over both halves: through shared memory, one 64-thread barrier per quadrant pair
      bars.xmax[hf][row] = mx;
      asm volatile("bar.sync %0, 64;" ::"r"(2 + q) : "memory");
      mx = fmaxf(mx, bars.xmax[hf ^ 1][row]);
      // the previous P V must be done before P is overwritten or O is rescaled
      if (ok && !mbar_wait(&bars.p_empty, (j & 1) ^ 1, abort_flag, status, KID_ATTN_PREFILL, 7)) ok = false;
      ok = __all_sync(0xffffffffu, ok);
      if (ok) {
      tc_fence_after();
      float alpha = 1.f;
      bool need = false;
      if (mx > m_ref + TC_RESCALE_THRESHOLD || (m_ref == -INFINITY && mx > -INFINITY)) {
        alpha = (m_ref == -INFINITY) ? 0.f : exp2f(m_ref - mx);
        m_ref = mx;
        need = j > 0;                              // O holds nothing before the first P V
      }
      if (__any_sync(0xffffffffu, need)) {
        // rescale this warp's half of the 32 lanes of O (lanes that did not move keep alpha = 1)
#pragma unroll
        for (int c = 0; c < TC_HD / 2; c += 16) {
          uint32_t r[16];
          tmem_ld_x16(tmem_o + lane_base + hf * (TC_HD / 2) + c, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
          tmem_st_x16(tmem_o + lane_base + hf * (TC_HD / 2) + c, r);
        }
        tmem_st_wait();
      }
      l_sum *= alpha;
      // P = 2^(s * scale - m_ref), BF16, into 128-byte-swizzled K-major shared memory: row `row`, 16-byte chunk c of 64-key
      // block kb (= this warp's half) at (row / 8) * 1024 + (row % 8) * 128 + ((c ^ (row % 8)) * 16)
      const float mr = (m_ref == -INFINITY) ? 0.f : m_ref;
      float ls4[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t pk[HB / 2];
#pragma unroll
      for (int i = 0; i < HB / 2; ++i) {
        // one FMA and one MUFU per value; a masked score is -inf and gives exactly 0
        const float p0 = ex2_approx(fmaf(sv[2 * i], scale_log2, -mr));
        const float p1 = ex2_approx(fmaf(sv[2 * i + 1], scale_log2, -mr));
        pk[i] = pack_bf16x2(p0, p1);
        ls4[i & 3] += p0 + p1;
      }
      // P stays in tensor memory: row = lane, two BF16 keys per 32-bit column, this warp's 64 keys = 32 columns; the second
      // product reads it from there as its A operand (no trip through shared memory, whose bandwidth the two products'
      // operand reads already use up)
      tmem_st_x16(tmem_p + lane_base + hf * (HB / 2), pk);
      tmem_st_x16(tmem_p + lane_base + hf * (HB / 2) + 16, pk + 16);
      tmem_st_wait();
      l_sum += (ls4[0] + ls4[1]) + (ls4[2] + ls4[3]);
      tc_fence_before();
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");
      if (e == 0 && ok) mbar_arrive(&bars.p_full);
    }
    if (ok) ok = mbar_wait(&bars.o_done, 0, abort_flag, status, KID_ATTN_PREFILL, 8);
    ok = __all_sync(0xffffffffu, ok);
    // the row's sum over both halves
    bars.xmax[hf][row] = l_sum;
    asm volatile("bar.sync %0, 64;" ::"r"(2 + q) : "memory");
    if (ok) {
      tc_fence_after();
      l_sum += bars.xmax[hf ^ 1][row];
      // learnable soft-max: one extra logit per head that enters the denominator only
      if (sinks != nullptr) l_sum += (m_ref == -INFINITY) ? 1.f : exp2f(sinks[h] * 1.4426950408889634f - m_ref);
      const float inv = l_sum > 0.f ? 1.f / l_sum : 0.f;
      __nv_bfloat16* orow = out + (size_t)(qs + r0 + row) * ldo + (size_t)h * TC_HD + hf * (TC_HD / 2);
#pragma unroll
      for (int c = 0; c < TC_HD / 2; c += 16) {
        uint32_t r[16];
        tmem_ld_x16(tmem_o + lane_base + hf * (TC_HD / 2) + c, r);
        tmem_ld_wait();
        if (live) {
          uint4 o0, o1;
          o0.x = pack_bf16x2(__uint_as_float(r[0]) * inv, __uint_as_float(r[1]) * inv);
          o0.y = pack_bf16x2(__uint_as_float(r[2]) * inv, __uint_as_float(r[3]) * inv);
          o0.z = pack_bf16x2(__uint_as_float(r[4]) * inv, __uint_as_float(r[5]) * inv);
          o0.w = pack_bf16x2(__uint_as_float(r[6]) * inv, __uint_as_float(r[7]) * inv);
          o1.x = pack_bf16x2(__uint_as_float(r[8]) * inv, __uint_as_float(r[9]) * inv);
          o1.y = pack_bf16x2(__uint_as_float(r[10]) * inv, __uint_as_float(r[11]) * inv);
          o1.z = pack_bf16x2(__uint_as_float(r[12]) * inv, __uint_as_float(r[13]) * inv);
          o1.w = pack_bf16x2(__uint_as_float(r[14]) * inv, __uint_as_float(r[15]) * inv);
          *reinterpret_cast<uint4*>(orow + c) = o0;
          *reinterpret_cast<uint4*>(orow + c + 8) = o1;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (bars.abort_flag) {
    const uint64_t t0w = globaltimer_ns();
    while (globaltimer_ns() - t0w < 200000ull) { __nanosleep(1000); }
  }
  if (warp == 1) { __syncwarp(); tc_fence_after(); tmem_dealloc(tmem_base, 512); }
}


// ------------------------------------------------------------------------------------------------
// Two CTAs per SM, 64-key tiles. The same products and masks, arranged so that two CTAs fit one SM and every role runs
// ahead of the next: per CTA 97 KB of shared memory (Q, two K tiles and two V tiles of one 64-key page each), 256 columns
// of tensor memory (two S buffers of 64 columns and O; P is written over the first 32 columns of the S buffer it came
// from, by the thread that owns the row, after it has taken its S values into registers), 6 warps (TMA, MMA, one softmax
// warp per lane quadrant, a thread owning a row). Q K(j+1)ᵀ is issued as soon as its K page is there, i.e. while the
// softmax warps are still on tile j; P V(j) runs while they are on tile j + 1; only the rare rescale of O waits for the
// previous P V. FF_ATTN_PREFILL_SPLIT=2 puts two softmax warps on every lane quadrant (32 columns each).
// Key heads of dk and value heads of dv elements (multiples of 16): Q Kᵀ runs dk / 16 steps, P V covers 64 or 128 columns;
// TMA fills the columns of a box that lie past the head with zeros.
// ------------------------------------------------------------------------------------------------
constexpr int T2_BN = 64;                                          // keys per tile = one cache page
constexpr int T2_KV_BYTES = T2_BN * TC_HD * 2;                     // 16 KiB
constexpr int TC2_SMEM = TC_Q_BYTES + 4 * T2_KV_BYTES + 1024;      // 97 KiB
constexpr int LAT_SMEM = 3 * (16384 + 2 * 8192) + 2 * T2_KV_BYTES + 1024;      // latent form: three 64-column blocks of Q and K, 129 KiB

// what a launch adds to plain causal attention over 128-wide heads
struct PrefillForm {
  int window, chunk, causal, dk, dv;
  int gated;                       // the result is multiplied by the sigmoid of a [rows, hq * dv] gate (tensor map tmG)
  int keep;                        // with a window: the first `keep` positions stay visible
  float cap_in;                    // CAP: score s becomes cap tanh(s / cap); cap_in = scale / cap
  const __nv_bfloat16* head_gate;  // the result of head h is multiplied by the sigmoid of head_gate[row * ldhg + h]
  int ldhg;
  // LAT: keys and values expanded from latents. The maps of K and V are over expanded rows [key rows, heads * dk | heads * dv]; page t of
  // sequence b is at key row (exp_off[b] + t) * 64. The last dr elements of queries and keys come from maps of their own: tmG, rows with
  // head h at column h * qr_pitch + qr_col, and tmR, the cache's rows, at column kr_col.
  const int* exp_off;
  int dr, qr_pitch, qr_col, kr_col;
};

// Capped scores. N raw products of a thread become tanh(y), y = s cap_in; the cap is the factor of the exponent. Where all |y| of the
// warp are at most 1 -- the usual case, caps being there for outliers -- tanh is a polynomial, two values per instruction, which
// leaves the special-function unit to the soft-max: y times a Chebyshev fit of tanh(y) / y in y^2 on [0, 1], error 5.5e-7.
// Otherwise 1 - 2 / (1 + e^(2y)).
template <int N>
__device__ __forceinline__ void cap_scores(float (&sv)[N], float cap_in) {
  float am[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < N; ++i) am[i & 3] = fmaxf(am[i & 3], fabsf(sv[i]));
  const float most = fmaxf(fmaxf(am[0], am[1]), fmaxf(am[2], am[3]));
  if (__all_sync(0xffffffffu, most * cap_in <= 1.0f)) {
    const uint64_t c = f2_pack(cap_in, cap_in);
    auto k = [](float v) { return f2_pack(v, v); };
    const uint64_t k0 = k(0.999999463558197f), k1 = k(-0.33329179883003235f), k2 = k(0.13282513618469238f), k3 = k(-0.05163545906543732f),
                   k4 = k(0.01677677594125271f), k5 = k(-0.0030804092530161142f);
#pragma unroll
    for (int i = 0; i < N; i += 2) {
      const uint64_t y = f2_mul(f2_pack(sv[i], sv[i + 1]), c), z = f2_mul(y, y);
      uint64_t r = f2_fma(k5, z, k4);
      r = f2_fma(r, z, k3);
      r = f2_fma(r, z, k2);
      r = f2_fma(r, z, k1);
      r = f2_fma(r, z, k0);
      f2_unpack(f2_mul(y, r), sv[i], sv[i + 1]);
    }
  } else {
    const float e = 2.0f * 1.4426950408889634f * cap_in;
#pragma unroll
    for (int i = 0; i < N; ++i) sv[i] = 1.0f - __fdividef(2.0f, 1.0f + ex2_approx(fminf(sv[i] * e, 100.0f)));
  }
}

// o * inv, times the sigmoid of the gate where there is one (`gate`: the row of a swizzled gate tile in shared memory, `sw` =
// row % 8, `chunk` its first 16-byte chunk); 16 columns, two 16-byte stores
__device__ __forceinline__ void store_o16(__nv_bfloat16* dst, const uint32_t* r, float inv, const uint8_t* gate, int chunk, int sw) {
  float v[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]) * inv;
  if (gate != nullptr) {
    const uint4 g0 = *reinterpret_cast<const uint4*>(gate + ((chunk ^ sw) << 4)), g1 = *reinterpret_cast<const uint4*>(gate + (((chunk + 1) ^ sw) << 4));
    const uint32_t gw[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float2 g = unpack_bf16x2(gw[i]);
      v[2 * i] = __fdividef(v[2 * i], 1.0f + __expf(-g.x));
      v[2 * i + 1] = __fdividef(v[2 * i + 1], 1.0f + __expf(-g.y));
    }
  }
  uint32_t o[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) o[i] = pack_bf16x2(v[2 * i], v[2 * i + 1]);
  reinterpret_cast<uint4*>(dst)[0] = make_uint4(o[0], o[1], o[2], o[3]);
  reinterpret_cast<uint4*>(dst)[1] = make_uint4(o[4], o[5], o[6], o[7]);
}

struct alignas(8) Tc2Bars {
  uint64_t q_full, g_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2], p_full[2], pv_done[2];
  uint32_t tmem_base;
  int abort_flag;
  float xmax[2][TC_BM];
};

// WIDE: heads are exactly 128 wide; EXTRA: the launch may have a block-local mask, kept first positions or a gate (plain launches keep
// an instance with none of them); CAP: scores are capped; LAT: latent attention over expanded keys and values, heads of up to 128 + 64
// elements (one CTA per SM).
template <int SPLIT, bool WIDE, bool EXTRA, bool CAP, bool LAT = false>
__global__ void __launch_bounds__(64 + 128 * SPLIT, LAT ? 1 : 2)
attn_prefill_tc2_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                        const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmG, const __grid_constant__ CUtensorMap tmR,
                        const int* __restrict__ block_table, const int* __restrict__ q_start, const int* __restrict__ q_lens,
                        const int* __restrict__ ctx_lens, __nv_bfloat16* __restrict__ out, int hq, int hkv, int ldo,
                        int max_blocks, int num_blocks, float scale_log2, const PrefillForm f, int* status,
                        const float* __restrict__ sinks) {
  const int b = blockIdx.z, h = blockIdx.y;
  const int qlen = q_lens[b];
  const int r0 = (gridDim.x - 1 - blockIdx.x) * TC_BM;            // long (late) query tiles first
  if (r0 >= qlen) return;
  extern __shared__ uint8_t smem_raw[];
  __shared__ Tc2Bars bars;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int BLOCKS = LAT ? 3 : 2;                              // 64-column blocks of a Q and a K tile
  constexpr int K_BYTES = BLOCKS * 8192;
  uint8_t* sQ = smem;
  uint8_t* sK = smem + BLOCKS * 16384;                             // two K tiles, then two V tiles
  uint8_t* sV = sK + 2 * K_BYTES;
  const int ctx = ctx_lens[b], qs = q_start[b];
  const int kvh = h / (hq / hkv);
  const int past = ctx - qlen;
  const int real = min(TC_BM, qlen - r0);
  const int causal = f.causal, window = f.window, chunk = EXTRA ? f.chunk : 0, dk = WIDE ? TC_HD : f.dk, dv = WIDE ? TC_HD : f.dv;
  const bool gated = EXTRA && f.gated != 0;
  const bool k_hi = dk > 64, v_hi = dv > 64;                       // heads up to 64 wide: the upper 64 columns are not loaded
  auto first_visible = [&](int pos) { return window > 0 ? max(0, pos - window + 1) : (chunk > 0 ? pos / chunk * chunk : 0); };
  const int last_key = causal ? past + r0 + real - 1 : ctx - 1;
  const int first_key = first_visible(past + r0);
  const int t0 = first_key / T2_BN, t1 = last_key / T2_BN + 1;
  // kept first positions in pages before the window's first: those pages come as the first tiles
  const int keep = EXTRA ? f.keep : 0;
  const int tkeep = EXTRA ? min(t0, (keep + T2_BN - 1) / T2_BN) : 0;
  const int ntiles = t1 - t0 + tkeep;
  auto tile_page = [&](int j) { return EXTRA && j < tkeep ? j : t0 + j - tkeep; };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
    mbar_init(&bars.q_full, 1); mbar_init(&bars.g_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars.k_full[i], 1); mbar_init(&bars.k_empty[i], 1); mbar_init(&bars.v_full[i], 1); mbar_init(&bars.v_empty[i], 1);
      mbar_init(&bars.s_full[i], 1); mbar_init(&bars.p_full[i], 1); mbar_init(&bars.pv_done[i], 1);
    }
    bars.abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(&bars.tmem_base, 256); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = bars.tmem_base;          // S buffer i: columns 64 i .. 64 i + 63; its P over the first 32 of them
  const uint32_t tmem_o = bars.tmem_base + 128;
  volatile int* abort_flag = &bars.abort_flag;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(&bars.q_full, (k_hi ? TC_Q_BYTES : TC_Q_BYTES / 2) + (LAT ? 16384 : 0));
      tma_load_2d(sQ, &tmQ, &bars.q_full, h * dk, qs + r0);
      if (LAT) tma_load_2d(sQ + 2 * TC_BM * 128, &tmG, &bars.q_full, h * f.qr_pitch + f.qr_col, qs + r0);
      if (k_hi) tma_load_2d(sQ + TC_BM * 128, &tmQ, &bars.q_full, h * dk + 64, qs + r0);
      bool ok = true, bad = false;
      const int nblk = (ctx + TC_PAGE - 1) / TC_PAGE;
      auto tile_row = [&](int j) -> int {
        int page = tile_page(j);
        if (page >= nblk) page = nblk - 1;                   // past the context: any valid page, its keys are masked
        int blk = block_table[(size_t)b * max_blocks + page];
        if (blk < 0 || blk >= num_blocks) { bad = true; blk = 0; }
        return (blk * hkv + (LAT ? 0 : kvh)) * TC_PAGE;
      };
      const int exp0 = LAT ? f.exp_off[b] : 0;
      // a tile: block d0 = [64 keys x 64 d] (8 KiB), then block d1. K runs one tile ahead of V: K(j + 1) is free once
      // Q K(j - 1) has run, V(j) only once P V(j - 2) has.
      auto load_k = [&](int j) -> bool {
        const int st = j & 1; const uint32_t ph = (j >> 1) & 1;
        const int row = tile_row(j);
        if (!mbar_wait(&bars.k_empty[st], ph ^ 1, abort_flag, status, KID_ATTN_PREFILL, 21)) return false;
        mbar_expect_tx(&bars.k_full[st], (k_hi ? T2_KV_BYTES : T2_KV_BYTES / 2) + (LAT ? 8192 : 0));
        const int kx = LAT ? h * dk : 0, ky = LAT ? (exp0 + tile_page(j)) * TC_PAGE : row;
        tma_load_2d(sK + st * K_BYTES, &tmK, &bars.k_full[st], kx, ky);
        if (k_hi) tma_load_2d(sK + st * K_BYTES + 8192, &tmK, &bars.k_full[st], kx + 64, ky);
        if (LAT) tma_load_2d(sK + st * K_BYTES + 16384, &tmR, &bars.k_full[st], f.kr_col, row);
        return true;
      };
      ok = load_k(0);
      for (int j = 0; j < ntiles && ok; ++j) {
        if (j + 1 < ntiles && !load_k(j + 1)) { ok = false; break; }
        const int st = j & 1; const uint32_t ph = (j >> 1) & 1;
        const int row = LAT ? (exp0 + tile_page(j)) * TC_PAGE : tile_row(j), vx = LAT ? h * dv : 0;
        if (!mbar_wait(&bars.v_empty[st], ph ^ 1, abort_flag, status, KID_ATTN_PREFILL, 22)) { ok = false; break; }
        mbar_expect_tx(&bars.v_full[st], v_hi ? T2_KV_BYTES : T2_KV_BYTES / 2);
        tma_load_2d(sV + st * T2_KV_BYTES, &tmV, &bars.v_full[st], vx, row);
        if (v_hi) tma_load_2d(sV + st * T2_KV_BYTES + 8192, &tmV, &bars.v_full[st], vx + 64, row);
      }
      if (ok && gated) {
        // the gate tile takes the place of Q once the last Q Kᵀ has read it; it arrives under the last soft-max and P V
        const int st = (ntiles - 1) & 1;
        if (mbar_wait(&bars.k_empty[st], ((ntiles - 1) >> 1) & 1, abort_flag, status, KID_ATTN_PREFILL, 31)) {
          mbar_expect_tx(&bars.g_full, v_hi ? TC_Q_BYTES : TC_Q_BYTES / 2);
          tma_load_2d(sQ, &tmG, &bars.g_full, h * dv, qs + r0);
          if (v_hi) tma_load_2d(sQ + TC_BM * 128, &tmG, &bars.g_full, h * dv + 64, qs + r0);
        }
      }
      if (bad) set_status(status, KID_ATTN_PREFILL, FF_ERR_BOUNDS, b, r0 / TC_BM);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc(1, 1, 0, 0, TC_BM, T2_BN);
      const uint32_t idesc_o = umma_idesc(1, 1, 0, 1, TC_BM, v_hi ? TC_HD : TC_HD / 2);
      const int ksteps = dk >> 4;
      const uint32_t q_addr = smem_u32(sQ);
      bool ok = mbar_wait(&bars.q_full, 0, abort_flag, status, KID_ATTN_PREFILL, 23);
      auto issue_s = [&](int j) -> bool {
        const int st = j & 1; const uint32_t ph = (j >> 1) & 1;
        if (!mbar_wait(&bars.k_full[st], ph, abort_flag, status, KID_ATTN_PREFILL, 24)) return false;
        // this S buffer still holds the P of tile j - 2: that tile's P V has to be complete
        if (j >= 2 && !mbar_wait(&bars.pv_done[st], ph ^ 1, abort_flag, status, KID_ATTN_PREFILL, 25)) return false;
        tc_fence_after();
        const uint32_t k_addr = smem_u32(sK + st * K_BYTES);
        if (LAT) {
          const int rsteps = f.dr >> 4;
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            if (k >= rsteps) break;
            umma_f16(tmem_s + st * T2_BN, umma_desc_sw128(q_addr + 2 * 16384 + k * 32, 16, 1024), umma_desc_sw128(k_addr + 2 * 8192 + k * 32, 16, 1024),
                     idesc_s, k != 0);
          }
        }
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          if (k >= ksteps) break;
          // Q: 64-column block k / 4 of a 128-row tile (16 KiB), 32 bytes per k-step; K: the same with 64 rows (8 KiB)
          umma_f16(tmem_s + st * T2_BN, umma_desc_sw128(q_addr + (k >> 2) * 16384 + (k & 3) * 32, 16, 1024),
                   umma_desc_sw128(k_addr + (k >> 2) * 8192 + (k & 3) * 32, 16, 1024), idesc_s, LAT || k != 0);
        }
        umma_commit(&bars.s_full[st]);
        umma_commit(&bars.k_empty[st]);
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; j < ntiles && ok; ++j) {
        if (j + 1 < ntiles) { ok = issue_s(j + 1); if (!ok) break; }
        const int st = j & 1; const uint32_t ph = (j >> 1) & 1;
        if (!mbar_wait(&bars.p_full[st], ph, abort_flag, status, KID_ATTN_PREFILL, 26)) { ok = false; break; }
        if (!mbar_wait(&bars.v_full[st], ph, abort_flag, status, KID_ATTN_PREFILL, 27)) { ok = false; break; }
        tc_fence_after();
        const uint32_t v_addr = smem_u32(sV + st * T2_KV_BYTES);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          // P: 16 keys = 8 columns of packed pairs; V: 16 key rows = 2 KiB inside each 64-dim block, blocks 8 KiB apart
          umma_f16_ts(tmem_o, tmem_s + st * T2_BN + k * 8, umma_desc_sw128(v_addr + k * 2048, 8192, 1024), idesc_o,
                      (j > 0) || (k != 0));
        }
        umma_commit(&bars.pv_done[st]);
        umma_commit(&bars.v_empty[st]);
      }
    }
  } else {
    constexpr int HB = T2_BN / SPLIT;             // columns of a tile per thread
    const int q = warp & 3;
    const int hf = (warp - 2) >> 2;
    const int row = q * 32 + lane;
    const int e = (warp - 2) * 32 + lane;
    const bool live = row < real;
    const int pos = past + r0 + row;
    const int hi = live ? (causal ? pos : ctx - 1) : -1;
    const int lo = live ? first_visible(pos) : 0;
    float m_ref = -INFINITY, l_sum = 0.f;
    bool ok = true;
    const uint32_t lane_base = (uint32_t(q * 32) << 16);
    const int tile_hi_min = causal ? past + r0 : ctx - 1;
    const int tile_lo_max = first_visible(past + r0 + real - 1);
    for (int j = 0; j < ntiles; ++j) {
      const int st = j & 1; const uint32_t ph = (j >> 1) & 1;
      if (ok && !mbar_wait(&bars.s_full[st], ph, abort_flag, status, KID_ATTN_PREFILL, 28)) ok = false;
      ok = __all_sync(0xffffffffu, ok);
      float sv[HB];
      float mx = -INFINITY;
      const uint32_t s_addr = tmem_s + lane_base + st * T2_BN;
      if (ok) {
        tc_fence_after();
        {
          uint32_t r[HB];
          if (HB == 64) { tmem_ld_x32(s_addr, r); tmem_ld_x32(s_addr + 32, r + 32); }
          else tmem_ld_x32(s_addr + hf * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < HB; ++i) sv[i] = __uint_as_float(r[i]);
        }
        const int tile0 = tile_page(j) * T2_BN, k0 = tile0 + hf * HB;
        if (CAP) cap_scores<HB>(sv, f.cap_in);
        float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
        if ((tile0 >= tile_lo_max || (EXTRA && tile0 + T2_BN <= keep)) && tile0 + T2_BN - 1 <= tile_hi_min) {
#pragma unroll
          for (int i = 0; i < HB; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], sv[i]);
        } else {
#pragma unroll
          for (int i = 0; i < HB; ++i) {
            const int key = k0 + i;
            const float t = ((key >= lo || (EXTRA && key < keep)) && key <= hi) ? sv[i] : -INFINITY;
            sv[i] = t;
            mx4[i & 3] = fmaxf(mx4[i & 3], t);
          }
        }
        mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale_log2;
      }
      if (SPLIT == 2) {
        // after this barrier both warps of the pair hold their S columns in registers: P may overwrite S
        bars.xmax[hf][row] = mx;
        asm volatile("bar.sync %0, 64;" ::"r"(2 + q) : "memory");
        mx = fmaxf(mx, bars.xmax[hf ^ 1][row]);
      }
      float alpha = 1.f;
      bool need = false;
      if (ok && (mx > m_ref + TC_RESCALE_THRESHOLD || (m_ref == -INFINITY && mx > -INFINITY))) {
        alpha = (m_ref == -INFINITY) ? 0.f : exp2f(m_ref - mx);
        m_ref = mx;
        need = j > 0;
      }
      if (__any_sync(0xffffffffu, need)) {
        // O is rescaled in place: the P V of the previous tile has to be complete (the rare path)
        if (ok && !mbar_wait(&bars.pv_done[st ^ 1], ((j - 1) >> 1) & 1, abort_flag, status, KID_ATTN_PREFILL, 30)) ok = false;
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
          tc_fence_after();
#pragma unroll
          for (int c = 0; c < TC_HD / SPLIT; c += 16) {
            if (hf * (TC_HD / SPLIT) + c >= dv) break;
            uint32_t r[16];
            tmem_ld_x16(tmem_o + lane_base + hf * (TC_HD / SPLIT) + c, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
            tmem_st_x16(tmem_o + lane_base + hf * (TC_HD / SPLIT) + c, r);
          }
          tmem_st_wait();
        }
      }
      if (ok) {
        l_sum *= alpha;
        const float mr = (m_ref == -INFINITY) ? 0.f : m_ref;
        float ls4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int c = 0; c < HB / 2; c += 16) {
          uint32_t pk[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const float p0 = ex2_approx(fmaf(sv[2 * (c + i)], scale_log2, -mr));
            const float p1 = ex2_approx(fmaf(sv[2 * (c + i) + 1], scale_log2, -mr));
            pk[i] = pack_bf16x2(p0, p1);
            ls4[i & 3] += p0 + p1;
          }
          // P over the first 32 columns of this S buffer: the thread's own lane, whose S values are in registers by now
          tmem_st_x16(s_addr + hf * (HB / 2) + c, pk);
        }
        tmem_st_wait();
        l_sum += (ls4[0] + ls4[1]) + (ls4[2] + ls4[3]);
        tc_fence_before();
      }
      // one arrival for the whole tile; an arrival per warp (no common barrier) measured 1.5 % slower
      if (SPLIT == 2) asm volatile("bar.sync 1, 256;" ::: "memory");
      else asm volatile("bar.sync 1, 128;" ::: "memory");
      if (e == 0 && ok) mbar_arrive(&bars.p_full[st]);
    }
    // the last P V
    if (ok && !mbar_wait(&bars.pv_done[(ntiles - 1) & 1], ((ntiles - 1) >> 1) & 1, abort_flag, status, KID_ATTN_PREFILL, 29)) ok = false;
    if (ok && gated && !mbar_wait(&bars.g_full, 0, abort_flag, status, KID_ATTN_PREFILL, 32)) ok = false;
    ok = __all_sync(0xffffffffu, ok);
    if (SPLIT == 2) {
      bars.xmax[hf][row] = l_sum;
      asm volatile("bar.sync %0, 64;" ::"r"(2 + q) : "memory");
      l_sum += bars.xmax[hf ^ 1][row];
    }
    if (ok) {
      tc_fence_after();
      if (sinks != nullptr) l_sum += (m_ref == -INFINITY) ? 1.f : exp2f(sinks[h] * 1.4426950408889634f - m_ref);
      float inv = l_sum > 0.f ? 1.f / l_sum : 0.f;
      if (EXTRA && f.head_gate != nullptr && live)
        inv = __fdividef(inv, 1.0f + __expf(-__bfloat162float(f.head_gate[(size_t)(qs + r0 + row) * f.ldhg + h])));
      __nv_bfloat16* orow = out + (size_t)(qs + r0 + row) * ldo + (size_t)h * dv + hf * (TC_HD / SPLIT);
#pragma unroll
      for (int c = 0; c < TC_HD / SPLIT; c += 16) {
        if (hf * (TC_HD / SPLIT) + c >= dv) break;
        uint32_t r[16];
        tmem_ld_x16(tmem_o + lane_base + hf * (TC_HD / SPLIT) + c, r);
        tmem_ld_wait();
        const int col = hf * (TC_HD / SPLIT) + c;                       // gate tile: 64-column halves of [128 rows][128 bytes]
        if (live) store_o16(orow + c, r, inv, gated ? sQ + (col >> 6) * (TC_BM * 128) + row * 128 : nullptr, (col & 63) >> 3, row & 7);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (bars.abort_flag) {
    const uint64_t t0w = globaltimer_ns();
    while (globaltimer_ns() - t0w < 200000ull) { __nanosleep(1000); }
  }
  if (warp == 1) { __syncwarp(); tc_fence_after(); tmem_dealloc(bars.tmem_base, 256); }
}

}  // namespace ff
using namespace ff;

// Same contract as ff_attn_prefill (attention_paged.cu). q: packed rows [rows, ldq] with head h at columns h*dk;
// out rows 16-byte aligned (ldo % 8 == 0). window > 0 sliding, 0 causal, < 0 bidirectional; chunk > 0: a query sees the keys
// of its own block of `chunk` positions that are not after it. dk / dv: widths of the key and value heads (multiples of 16,
// at most 128); ldv: pitch of the value cache's rows (dv, or the key rows' width where the values are their first columns). gate:
// optional [rows, hq * dv] with row pitch ldg, 16-byte aligned. keep: with a window, the first `keep` positions stay visible.
// softcap > 0: scores become softcap tanh(score / softcap). head_gate: optional [rows, hq] with row pitch ldhg.
FF_EXPORT int ff_attn_prefill_tc(const void* q, const void* kcache, const void* vcache, const int* block_table,
                                 const int* q_start, const int* q_lens, const int* ctx_lens, void* out, int batch,
                                 int total_rows, int max_q_len, int hq, int hkv, int dk, int dv, int ldq, int ldo,
                                 int max_blocks, int num_blocks, float scale, int window, int chunk, const float* sinks,
                                 const void* gate, int ldg, int ldv, int keep, float softcap, const void* head_gate, int ldhg, int* status,
                                 cudaStream_t s) {
  if (ldv < dv || ldv % 8 || keep < 0 || !(softcap >= 0.f) || (softcap > 0.f && sinks != nullptr)) return FF_HOST_BAD_SHAPE;
  if (batch <= 0 || max_q_len <= 0 || hq <= 0 || hkv <= 0 || hq % hkv || total_rows <= 0) return FF_HOST_BAD_SHAPE;
  if (dk < 16 || dk > TC_HD || dk % 16 || dv < 16 || dv > TC_HD || dv % 16 || chunk < 0 || !(scale > 0.f)) return FF_HOST_BAD_SHAPE;
  if (chunk > 0 && window != 0) return FF_HOST_UNSUPPORTED;
  if (ldq % 8 || ldo % 8 || (reinterpret_cast<uintptr_t>(out) & 15)) return FF_HOST_BAD_ALIGN;
  if (gate != nullptr && (ldg % 8 || (reinterpret_cast<uintptr_t>(gate) & 15))) return FF_HOST_BAD_ALIGN;
  CUtensorMap tmQ, tmK, tmV;
  if (int r = make_tmap_2d(&tmQ, q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (uint64_t)ldq, (uint64_t)total_rows,
                           (uint64_t)ldq * 2, 64, TC_BM)) return r;
  const uint64_t cache_rows = (uint64_t)num_blocks * hkv * TC_PAGE;
  if (int r = make_tmap_2d(&tmK, kcache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, dk, cache_rows, dk * 2, 64, TC_PAGE)) return r;
  if (int r = make_tmap_2d(&tmV, vcache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, dv, cache_rows, (uint64_t)ldv * 2, 64, TC_PAGE)) return r;
  const float scale_log2 = (softcap > 0.f ? softcap : scale) * 1.4426950408889634f;
  dim3 grid((max_q_len + TC_BM - 1) / TC_BM, hq, batch);
  const PrefillForm f = {window < 0 ? 0 : window, chunk, window < 0 ? 0 : 1, dk, dv, gate != nullptr ? 1 : 0, window > 0 ? keep : 0,
                         softcap > 0.f ? scale / softcap : 0.f, (const __nv_bfloat16*)head_gate, ldhg, nullptr, 0, 0, 0, 0};
  CUtensorMap tmG = tmQ;
  if (gate != nullptr)
    if (int r = make_tmap_2d(&tmG, gate, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (uint64_t)hq * dv, (uint64_t)total_rows, (uint64_t)ldg * 2, 64, TC_BM)) return r;
  // FF_ATTN_PREFILL_CTAS = 1 selects the one-CTA-per-SM kernel (deep K / V rings, eight softmax warps; plain 128-wide heads
  // only); the default is the two-CTAs-per-SM kernel
  static int two = -1;
  if (two < 0) { const char* e = getenv("FF_ATTN_PREFILL_CTAS"); two = (e != nullptr && e[0] == '1') ? 0 : TC_TWO_CTAS_DEFAULT; }
  const bool wide = dk == TC_HD && dv == TC_HD, extra = chunk > 0 || gate != nullptr || f.keep > 0 || head_gate != nullptr, cap = softcap > 0.f;
  if (two || extra || cap || !wide) {
    // FF_ATTN_PREFILL_SPLIT = 2: two softmax warps per lane quadrant (64 columns each) instead of one
    static int split = -1;
    if (split < 0) { const char* e = getenv("FF_ATTN_PREFILL_SPLIT"); split = (e != nullptr && (e[0] == '1' || e[0] == '2')) ? e[0] - '0' : TC2_SPLIT_DEFAULT; }
    auto go = [&](auto kern, int threads) -> int {
      if (int r = opt_in_smem(kern, TC2_SMEM)) return r;
      kern<<<grid, threads, TC2_SMEM, s>>>(tmQ, tmK, tmV, tmG, tmQ, block_table, q_start, q_lens, ctx_lens, (__nv_bfloat16*)out, hq, hkv, ldo,
                                           max_blocks, num_blocks, scale_log2, f, status, sinks);
      return launch_result();
    };
    if (!wide) return cap ? go(attn_prefill_tc2_kernel<1, false, true, true>, 192) : go(attn_prefill_tc2_kernel<1, false, true, false>, 192);
    if (cap) return extra ? go(attn_prefill_tc2_kernel<1, true, true, true>, 192) : go(attn_prefill_tc2_kernel<1, true, false, true>, 192);
    if (split == 2) return extra ? go(attn_prefill_tc2_kernel<2, true, true, false>, 320) : go(attn_prefill_tc2_kernel<2, true, false, false>, 320);
    return extra ? go(attn_prefill_tc2_kernel<1, true, true, false>, 192) : go(attn_prefill_tc2_kernel<1, true, false, false>, 192);
  }
  if (int r = opt_in_smem(attn_prefill_tc_kernel, TC_SMEM)) return r;
  attn_prefill_tc_kernel<<<grid, 320, TC_SMEM, s>>>(tmQ, tmK, tmV, block_table, q_start, q_lens, ctx_lens,
                                                    (__nv_bfloat16*)out, hq, hkv, ldo, max_blocks, num_blocks, scale_log2,
                                                    f.window, f.causal, status, sinks);
  return launch_result();
}

// Latent attention over keys and values expanded from the latents (prefill; one product of all heads' matrices with the rows the queries
// can see): head h's key is [expanded key (dk) | rotated key of the cache row (dr)]. q: rows [rows, ldq] with head h's unrotated part at
// column h * dk; q_rot: rows of heads * qr_pitch columns with its rotated part at h * qr_pitch + qr_col; expanded: [exp_rows, lde], head
// h's key at column h * dk and its value at hq * dk + h * dv; page t of sequence b starts at row (exp_off[b] + t) * 64; cache:
// [num_blocks, 1, 64, cache_width] with the rotated key at column kr_col. out [rows, ldo]. dk, dv multiples of 16 up to 128, dr up to 64.
FF_EXPORT int ff_attn_prefill_latent(const void* q, const void* q_rot, const void* expanded, const void* cache, const int* block_table,
                                     const int* q_start, const int* q_lens, const int* ctx_lens, const int* exp_off, void* out, int batch,
                                     int total_rows, int max_q_len, int hq, int dk, int dr, int dv, int ldq, int qr_pitch, int qr_col, int lde,
                                     int exp_rows, int cache_width, int kr_col, int ldo, int max_blocks, int num_blocks, float scale, int window,
                                     const void* head_gate, int ldhg, int* status, cudaStream_t s) {
  if (batch <= 0 || max_q_len <= 0 || hq <= 0 || total_rows <= 0 || exp_rows <= 0 || window < 0 || !(scale > 0.f)) return FF_HOST_BAD_SHAPE;
  if (dk < 16 || dk > TC_HD || dk % 16 || dv < 16 || dv > TC_HD || dv % 16 || dr < 16 || dr > 64 || dr % 16) return FF_HOST_BAD_SHAPE;
  if (ldq < hq * dk || lde < hq * (dk + dv) || qr_pitch < qr_col + dr || cache_width < kr_col + dr || exp_off == nullptr) return FF_HOST_BAD_SHAPE;
  if (ldq % 8 || lde % 8 || qr_pitch % 8 || qr_col % 8 || cache_width % 8 || kr_col % 8 || ldo % 8 || (reinterpret_cast<uintptr_t>(out) & 15)) return FF_HOST_BAD_ALIGN;
  constexpr auto BF = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  CUtensorMap tmQ, tmG, tmK, tmV, tmR;
  if (int r = make_tmap_2d(&tmQ, q, BF, 2, (uint64_t)hq * dk, total_rows, (uint64_t)ldq * 2, 64, TC_BM)) return r;
  if (int r = make_tmap_2d(&tmG, q_rot, BF, 2, (uint64_t)hq * qr_pitch, total_rows, (uint64_t)hq * qr_pitch * 2, 64, TC_BM)) return r;
  if (int r = make_tmap_2d(&tmK, expanded, BF, 2, (uint64_t)hq * dk, exp_rows, (uint64_t)lde * 2, 64, TC_PAGE)) return r;
  const __nv_bfloat16* values = (const __nv_bfloat16*)expanded + (size_t)hq * dk;
  if (int r = make_tmap_2d(&tmV, values, BF, 2, (uint64_t)hq * dv, exp_rows, (uint64_t)lde * 2, 64, TC_PAGE)) return r;
  if (int r = make_tmap_2d(&tmR, cache, BF, 2, cache_width, (uint64_t)num_blocks * TC_PAGE, (uint64_t)cache_width * 2, 64, TC_PAGE)) return r;
  PrefillForm f = {};
  f.window = window; f.causal = 1; f.dk = dk; f.dv = dv; f.head_gate = (const __nv_bfloat16*)head_gate; f.ldhg = ldhg;
  f.exp_off = exp_off; f.dr = dr; f.qr_pitch = qr_pitch; f.qr_col = qr_col; f.kr_col = kr_col;
  auto kern = dk == TC_HD && dv == TC_HD ? attn_prefill_tc2_kernel<2, true, true, false, true> : attn_prefill_tc2_kernel<2, false, true, false, true>;
  if (int r = opt_in_smem(kern, LAT_SMEM)) return r;
  kern<<<dim3((max_q_len + TC_BM - 1) / TC_BM, hq, batch), 320, LAT_SMEM, s>>>(tmQ, tmK, tmV, tmG, tmR, block_table, q_start, q_lens, ctx_lens,
      (__nv_bfloat16*)out, hq, 1, ldo, max_blocks, num_blocks, scale * 1.4426950408889634f, f, status, nullptr);
  return launch_result();
}
