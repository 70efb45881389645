// Gated delta rule with a decay per key channel (delta.cu), prompts: 64 tokens at a time on tensor cores, BF16 rows, dk <= 128.
// With l_t the logarithms of the decays, G_t = l_1 + .. + l_t over the chunk and S_0 the state before it, the recurrence is
//     A[t, s] = beta_t sum_d k_t k_s e^{G_t - G_s}  (s < t)       P[t, s] = sum_d q_t k_s e^{G_t - G_s}  (s <= t)
//     T = (I + A)^-1      W = T diag(beta) (K e^G)      U = T diag(beta) V - W S_0
//     O = (Q e^G) S_0 + P U                             S <- e^{G_C} S_0 + (K e^{G_C - G})^T U
// Two kernels:
//   delta_parts : what does not depend on the state, all chunks side by side: W, T diag(beta) V, Q e^G, K e^{G_C - G}, P and e^{G_C} go
//                 to scratch in the form the second kernel's shared memory takes them.
//   delta_scan  : the chunks of a sequence in order, 64 value columns per CTA, the state in FP32 accumulator registers. The next
//                 chunk's tiles are on their way while a chunk is worked on.
// Nothing of the recurrence is cut to 8 bits: an FP32 operand x enters a product as two BF16 values, hi and x - hi, and a product of
// two such operands is three products (hi hi, hi lo, lo hi).
// Exponents: a chunk is cut into four blocks of 16 tokens. With R_i the value of G before block i, e^{G_t - G_s} = e^{G_t - R_i}
// e^{R_i - G_s} for t in block i and s in an earlier block: both factors at most 1. Inside a block the second factor grows, up to
// e^{R_i - G} at the block's end: a block whose decays sum up to more than 2^-CD_SPAN in some channel takes its pairs one by one.
#include "delta.cuh"
#include "host_util.h"
#include "mma_sync.cuh"

namespace ff {

constexpr int CD = 64;                // tokens of a chunk
constexpr int CD_BLOCK = 16;
constexpr float CD_SPAN = 100.f;      // log2
constexpr int CDC = CD / 8;           // 16-byte chunks of a 64-wide tile's row
constexpr int CD_VT = 128;            // value columns delta_parts takes at a time

__device__ __forceinline__ void cd_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cd_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cd_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// two neighbours as BF16 values and BF16 remainders
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x - h.x, y - h.y);
}

// Scratch of one (chunk, head): images of the second kernel's tiles, then U in the order of its accumulators.
template <int KP>
struct DeltaParts {
  uint8_t w[2][CD * KP * 2], q[2][CD * KP * 2], k[2][CD * KP * 2], p[2][CD * CD * 2];      // value, remainder
  float keep[KP];                                                                          // e^{G_C}
};
template <int KP> constexpr size_t delta_record(int dv) { return sizeof(DeltaParts<KP>) + (size_t)CD * ((dv + DL_TILE - 1) / DL_TILE * DL_TILE) * 4; }

// chunks c0 .. c0 + count - 1 of every sequence; the record of (sequence, chunk, head) is number (sequence * count + chunk - c0) * H + head
struct DeltaRound { uint8_t* scratch; int c0, count; };

// three products of split operands
__device__ __forceinline__ void mma3(float (&d)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
  ms_mma(d, ah, bh0, bh1);
  ms_mma(d, ah, bl0, bl1);
  ms_mma(d, al, bh0, bh1);
}

template <int KP>
struct PartsSmem {
  static constexpr int GP = KP + 4, XP = KP + 8, AP = CD + 1;
  float g[CD * GP];                   // log2 of the decays, summed up inside every block of 16
  float total[4][KP];                 // a block's sum
  __nv_bfloat16 kx[CD * XP];
  union { __nv_bfloat16 qx[CD * XP]; uint8_t v[CD * CD_VT * 2]; };
  union { float a[CD * AP]; uint8_t t1[2][CD * CD * 2]; };
  float t[CD * AP];
  float beta[CD], fk[CD], fq[CD];
  int wide[4];                        // the block's pairs go one by one
};
static_assert(sizeof(__nv_bfloat16) * CD * PartsSmem<64>::XP < CD * CD_VT * 2, "the union holds the larger");

// grid (chunks, heads, sequences), 256 threads
template <int KP>
__global__ void __launch_bounds__(256, 2)
delta_parts_kernel(const DeltaArgs<__nv_bfloat16> p, const DeltaRound rd) {
  pdl_trigger();
  pdl_wait();
  using SM = PartsSmem<KP>;
  extern __shared__ __align__(128) uint8_t cd_raw[];
  SM& sm = *reinterpret_cast<SM*>((reinterpret_cast<uintptr_t>(cd_raw) + 127) & ~uintptr_t(127));
  constexpr int GP = SM::GP, XP = SM::XP, AP = SM::AP, KCH = KP / 8;
  const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
  const int r0 = p.row_start[seq] + (rd.c0 + blockIdx.x) * CD, n = min(CD, p.row_start[seq + 1] - r0);
  if (n <= 0) return;
  const int H = p.heads, G = p.kv_heads, kh = h / (H / G), dk = p.dk, dv = p.dv;
  uint8_t* rec = rd.scratch + (((size_t)seq * rd.count + blockIdx.x) * H + h) * delta_record<KP>(dv);
  DeltaParts<KP>& out = *reinterpret_cast<DeltaParts<KP>*>(rec);
  float* u_out = reinterpret_cast<float*>(rec + sizeof(DeltaParts<KP>));

  // ---- the chunk's rows; past the end: no decay, nothing written (k = 0, beta = 0)
  const float rate = p.rate[h] * 1.4426950408889634f;
  for (int i = tid; i < CD * KP / 4; i += 256) {
    const int t = i / (KP / 4), c = (i - t * (KP / 4)) * 4;
    float l[4] = {0.f, 0.f, 0.f, 0.f};
    uint2 kk = make_uint2(0, 0), qq = kk;
    if (t < n && c < dk) {
      const __nv_bfloat16* xr = p.x + (size_t)(r0 + t) * p.ldx + c;
      qq = *reinterpret_cast<const uint2*>(xr + (size_t)kh * dk);
      kk = *reinterpret_cast<const uint2*>(xr + (size_t)(G + kh) * dk);
      float z[4], b[4];
      load4(p.decay + (size_t)(r0 + t) * p.ldd + (size_t)h * dk + c, z);
      load4(p.dt_bias + (size_t)h * dk + c, b);
#pragma unroll
      for (int j = 0; j < 4; ++j) l[j] = log_decay(z[j], b[j], rate);
    }
    store4(sm.g + t * GP + c, l);
    *reinterpret_cast<uint2*>(sm.kx + t * XP + c) = kk;
    *reinterpret_cast<uint2*>(sm.qx + t * XP + c) = qq;
  }
  if (tid < CD) {
    const bool on = tid < n;
    sm.beta[tid] = on ? sigmoid_f(to_float(p.beta[(size_t)(r0 + tid) * p.ldb + h])) : 0.f;
    sm.fq[tid] = on ? p.unit[(size_t)(r0 + tid) * 2 * G + kh] : 0.f;
    sm.fk[tid] = on ? p.unit[(size_t)(r0 + tid) * 2 * G + G + kh] : 0.f;
  }
  if (tid < 4) sm.wide[tid] = 0;
  __syncthreads();
  for (int i = tid; i < 4 * KP; i += 256) {                // sums inside a block of 16
    const int b = i / KP, c = i - b * KP;
    float run = 0.f;
    float* at = sm.g + b * CD_BLOCK * GP + c;
#pragma unroll
    for (int t = 0; t < CD_BLOCK; ++t) { run += at[t * GP]; at[t * GP] = run; }
    sm.total[b][c] = run;
    if (run < -CD_SPAN) sm.wide[b] = 1;
  }
  __syncthreads();

  // ---- A and P, one 16 x 16 block (i, j), j <= i, per warp at a time
  for (int unit = warp; unit < 10; unit += 8) {
    const int i = unit < 1 ? 0 : unit < 3 ? 1 : unit < 6 ? 2 : 3, j = unit - i * (i + 1) / 2;
    float kk[2][4], qk[2][4];
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int e = 0; e < 4; ++e) { kk[a][e] = 0.f; qk[a][e] = 0.f; }
    if (i == j && sm.wide[i]) {
      for (int d = 0; d < dk; ++d)
#pragma unroll
        for (int a = 0; a < 2; ++a)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int t = 16 * i + gq + 8 * (e >> 1), s = 16 * i + 8 * a + 2 * tq + (e & 1);
            if (s > t) continue;
            const float f = ex2(sm.g[t * GP + d] - sm.g[s * GP + d]) * to_float(sm.kx[s * XP + d]);
            kk[a][e] = fmaf(to_float(sm.kx[t * XP + d]), f, kk[a][e]);
            qk[a][e] = fmaf(to_float(sm.qx[t * XP + d]), f, qk[a][e]);
          }
    } else {
#pragma unroll 1
      for (int ks = 0; ks < KP / 16; ++ks) {
        uint32_t kh4[4], kl4[4], qh4[4], ql4[4];
#pragma unroll
        for (int a = 0; a < 4; ++a) {                      // rows g, g + 8; channels 2t, 2t + 8
          const int t = 16 * i + gq + 8 * (a & 1), d = 16 * ks + 2 * tq + 8 * (a >> 1);
          const float2 l = *reinterpret_cast<const float2*>(sm.g + t * GP + d);
          const float fx = ex2(l.x), fy = ex2(l.y);
          const float2 kv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm.kx + t * XP + d)), qv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm.qx + t * XP + d));
          split2(kv.x * fx, kv.y * fy, kh4[a], kl4[a]);
          split2(qv.x * fx, qv.y * fy, qh4[a], ql4[a]);
        }
#pragma unroll
        for (int a = 0; a < 2; ++a) {
          uint32_t bh[2], bl[2];
#pragma unroll
          for (int b = 0; b < 2; ++b) {
            const int s = 16 * j + 8 * a + gq, d = 16 * ks + 2 * tq + 8 * b;
            const float2 l = *reinterpret_cast<const float2*>(sm.g + s * GP + d);
            float ex = -l.x, ey = -l.y;
            for (int m = j; m < i; ++m) { const float2 w = *reinterpret_cast<const float2*>(sm.total[m] + d); ex += w.x; ey += w.y; }
            const float2 kv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm.kx + s * XP + d));
            split2(kv.x * ex2(ex), kv.y * ex2(ey), bh[b], bl[b]);
          }
          mma3(kk[a], kh4, kl4, bh[0], bh[1], bl[0], bl[1]);
          mma3(qk[a], qh4, ql4, bh[0], bh[1], bl[0], bl[1]);
        }
      }
    }
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = 16 * i + gq + 8 * e, s = 16 * j + 8 * a + 2 * tq;
        const float rk = sm.beta[t] * sm.fk[t], rq = sm.fq[t], f0 = sm.fk[s], f1 = sm.fk[s + 1];
        sm.a[t * AP + s] = s < t ? rk * f0 * kk[a][2 * e] : 0.f;
        sm.a[t * AP + s + 1] = s + 1 < t ? rk * f1 * kk[a][2 * e + 1] : 0.f;
        uint32_t hi, lo;
        split2(s <= t ? rq * f0 * qk[a][2 * e] : 0.f, s + 1 <= t ? rq * f1 * qk[a][2 * e + 1] : 0.f, hi, lo);
        const uint32_t at = ms_off(t, s >> 3, CDC) + (s & 7) * 2;
        *reinterpret_cast<uint32_t*>(out.p[0] + at) = hi;
        *reinterpret_cast<uint32_t*>(out.p[1] + at) = lo;
      }
  }
  // ---- Q e^G, K e^{G_C - G} and e^{G_C}
  for (int i = tid; i < CD * KP / 2; i += 256) {
    const int t = i / (KP / 2), c = (i - t * (KP / 2)) * 2, b = t / CD_BLOCK;
    const float2 l = *reinterpret_cast<const float2*>(sm.g + t * GP + c);
    float2 before = l, after = make_float2(-l.x, -l.y);
    for (int m = 0; m < 4; ++m) {
      const float2 w = *reinterpret_cast<const float2*>(sm.total[m] + c);
      if (m < b) { before.x += w.x; before.y += w.y; } else { after.x += w.x; after.y += w.y; }
    }
    const float2 kv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm.kx + t * XP + c)), qv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm.qx + t * XP + c));
    const float fq = sm.fq[t], fk = sm.fk[t];
    const uint32_t at = ms_off(t, c >> 3, KCH) + (c & 7) * 2;
    uint32_t hi, lo;
    split2(qv.x * fq * ex2(before.x), qv.y * fq * ex2(before.y), hi, lo);
    *reinterpret_cast<uint32_t*>(out.q[0] + at) = hi;
    *reinterpret_cast<uint32_t*>(out.q[1] + at) = lo;
    split2(kv.x * fk * ex2(after.x), kv.y * fk * ex2(after.y), hi, lo);
    *reinterpret_cast<uint32_t*>(out.k[0] + at) = hi;
    *reinterpret_cast<uint32_t*>(out.k[1] + at) = lo;
  }
  for (int c = tid; c < KP; c += 256) out.keep[c] = ex2((sm.total[0][c] + sm.total[1][c]) + (sm.total[2][c] + sm.total[3][c]));
  __syncthreads();

  // ---- T = (I + A)^-1: the diagonal blocks by substitution (a column per lane), the others from them, by distance from the diagonal
  if (warp < 4 && lane < 16) {
    const float* a = sm.a + (16 * warp) * AP + 16 * warp;
    float x[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      float v = r == lane ? 1.f : 0.f;
#pragma unroll
      for (int s = 0; s < r; ++s) v = fmaf(-a[r * AP + s], x[s], v);
      x[r] = v;
    }
#pragma unroll
    for (int r = 0; r < 16; ++r) sm.t[(16 * warp + r) * AP + 16 * warp + lane] = x[r];
  }
  __syncthreads();
  for (int dist = 1; dist < 4; ++dist) {
    // M = sum_k A_ik T_kj goes where T_ji would be (above the diagonal), then T_ij = -T_ii M
    for (int e = tid; e < (4 - dist) * 256; e += 256) {
      const int j = e >> 8, i = j + dist, r = (e >> 4) & 15, c = e & 15;
      float v = 0.f;
      for (int s = 16 * j; s < 16 * i; ++s) v = fmaf(sm.a[(16 * i + r) * AP + s], sm.t[s * AP + 16 * j + c], v);
      sm.t[(16 * j + r) * AP + 16 * i + c] = v;
    }
    __syncthreads();
    for (int e = tid; e < (4 - dist) * 256; e += 256) {
      const int j = e >> 8, i = j + dist, r = (e >> 4) & 15, c = e & 15;
      float v = 0.f;
#pragma unroll
      for (int s = 0; s < 16; ++s) v = fmaf(-sm.t[(16 * i + r) * AP + 16 * i + s], sm.t[(16 * j + s) * AP + 16 * i + c], v);
      sm.t[(16 * i + r) * AP + 16 * j + c] = v;
    }
    __syncthreads();
  }
  // ---- T diag(beta) as an operand (A is no longer needed), blocks on and below the diagonal; the first value columns
  for (int i = tid; i < CD * CD / 2; i += 256) {
    const int t = i / (CD / 2), s = (i - t * (CD / 2)) * 2;
    if (s / 16 > t / 16) continue;
    uint32_t hi, lo;
    split2(sm.t[t * AP + s] * sm.beta[s], sm.t[t * AP + s + 1] * sm.beta[s + 1], hi, lo);
    const uint32_t at = ms_off(t, s >> 3, CDC) + (s & 7) * 2;
    *reinterpret_cast<uint32_t*>(sm.t1[0] + at) = hi;
    *reinterpret_cast<uint32_t*>(sm.t1[1] + at) = lo;
  }
  __syncthreads();
  const uint32_t aT0 = smem_u32(sm.t1[0]), aT1 = smem_u32(sm.t1[1]), aV = smem_u32(sm.v);
  auto t_frag = [&](uint32_t base, int i, int ks, uint32_t (&a)[4]) {
    ms_ldsm4(base + ms_off(16 * i + (lane & 7) + (((lane >> 3) & 1) << 3), 2 * ks + (lane >> 4), CDC), a[0], a[1], a[2], a[3]);
  };
  // ---- -W: a warp takes 16 channels of all rows
  for (int ct = warp; ct < KP / 16; ct += 8) {
    uint32_t bh[4][2][2], bl[4][2][2];                     // [16 tokens][8 channels][k half]
#pragma unroll
    for (int ks = 0; ks < 4; ++ks)
#pragma unroll
      for (int a = 0; a < 2; ++a)
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          const int s = 16 * ks + 2 * tq + 8 * b, d = 16 * ct + 8 * a + gq;
          float before = 0.f;
#pragma unroll
          for (int m = 0; m < ks; ++m) before += sm.total[m][d];
          const float x = to_float(sm.kx[s * XP + d]) * sm.fk[s] * ex2(sm.g[s * GP + d] + before);
          const float y = to_float(sm.kx[(s + 1) * XP + d]) * sm.fk[s + 1] * ex2(sm.g[(s + 1) * GP + d] + before);
          split2(x, y, bh[ks][a][b], bl[ks][a][b]);
        }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
      for (int ks = 0; ks <= i; ++ks) {
        uint32_t th[4], tl[4];
        t_frag(aT0, i, ks, th);
        t_frag(aT1, i, ks, tl);
#pragma unroll
        for (int a = 0; a < 2; ++a) mma3(acc[a], th, tl, bh[ks][a][0], bh[ks][a][1], bl[ks][a][0], bl[ks][a][1]);
      }
#pragma unroll
      for (int a = 0; a < 2; ++a)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          uint32_t hi, lo;
          split2(-acc[a][2 * e], -acc[a][2 * e + 1], hi, lo);
          const uint32_t at = ms_off(16 * i + gq + 8 * e, 2 * ct + a, KCH) + 4 * tq;
          *reinterpret_cast<uint32_t*>(out.w[0] + at) = hi;
          *reinterpret_cast<uint32_t*>(out.w[1] + at) = lo;
        }
    }
  }
  // ---- T diag(beta) V: a warp takes 16 columns of all rows; stored in the order of the second kernel's accumulators
  for (int v0 = 0; v0 < dv; v0 += CD_VT) {
    __syncthreads();                                       // Q, then the previous columns, are no longer read
    for (int i = tid; i < CD * CD_VT / 8; i += 256) {
      const int t = i / (CD_VT / 8), c = i - t * (CD_VT / 8);
      uint4 x = make_uint4(0, 0, 0, 0);
      if (t < n && v0 + c * 8 < dv) x = *reinterpret_cast<const uint4*>(p.x + (size_t)(r0 + t) * p.ldx + (size_t)2 * G * dk + (size_t)h * dv + v0 + c * 8);
      *reinterpret_cast<uint4*>(sm.v + ms_off(t, c, CD_VT / 8)) = x;
    }
    __syncthreads();
    const int col = v0 + 16 * warp;
    if (col >= (dv + DL_TILE - 1) / DL_TILE * DL_TILE) continue;
    float* dst = u_out + (size_t)(col / DL_TILE) * CD * DL_TILE;
    const int half = (col % DL_TILE) / 32, nt0 = (col % 32) / 8;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
      for (int ks = 0; ks <= i; ++ks) {
        uint32_t th[4], tl[4], b0, b1, b2, b3;
        t_frag(aT0, i, ks, th);
        t_frag(aT1, i, ks, tl);
        ms_ldsm4t(aV + ms_off(ks * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), 2 * warp + (lane >> 4), CD_VT / 8), b0, b1, b2, b3);
        ms_mma(acc[0], th, b0, b1); ms_mma(acc[0], tl, b0, b1);
        ms_mma(acc[1], th, b2, b3); ms_mma(acc[1], tl, b2, b3);
      }
#pragma unroll
      for (int a = 0; a < 2; ++a) store4(dst + ((size_t)((half * 4 + i) * 4 + nt0 + a) * 32 + lane) * 4, acc[a]);
    }
  }
}

template <int KP>
struct ScanSmem {
  uint8_t w[2][CD * KP * 2], q[2][CD * KP * 2], k[2][CD * KP * 2], p[2][CD * CD * 2];
  uint8_t s[2][KP * DL_TILE * 2];     // operand copy of the state
  uint8_t u[2][CD * DL_TILE * 2];
};

// acc += A B, both split; A row-major tile from row m0, B [k][n] rows from column n0
template <int NT>
__device__ __forceinline__ void product3(float (&acc)[NT][4], uint32_t a0, uint32_t a1, int a_chunks, int m0, uint32_t b0, uint32_t b1, int n0, int ksteps, int lane) {
#pragma unroll 2
  for (int ks = 0; ks < ksteps; ++ks) {
    uint32_t ah[4], al[4];
    const uint32_t ao = ms_off(m0 + (lane & 7) + (((lane >> 3) & 1) << 3), 2 * ks + (lane >> 4), a_chunks);
    ms_ldsm4(a0 + ao, ah[0], ah[1], ah[2], ah[3]);
    ms_ldsm4(a1 + ao, al[0], al[1], al[2], al[3]);
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) {
      uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
      const uint32_t bo = ms_off(ks * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), (n0 >> 3) + 2 * np + (lane >> 4), CDC);
      ms_ldsm4t(b0 + bo, h0, h1, h2, h3);
      ms_ldsm4t(b1 + bo, l0, l1, l2, l3);
      mma3(acc[2 * np], ah, al, h0, h1, l0, l1);
      mma3(acc[2 * np + 1], ah, al, h2, h3, l2, l3);
    }
  }
}

// grid (value tiles, heads, sequences), 256 threads
template <int KP>
__global__ void __launch_bounds__(256, 1)
delta_scan_kernel(const DeltaArgs<__nv_bfloat16> p, const DeltaRound rd) {
  pdl_trigger();
  pdl_wait();
  using SM = ScanSmem<KP>;
  extern __shared__ __align__(128) uint8_t cd_raw[];
  SM& sm = *reinterpret_cast<SM*>((reinterpret_cast<uintptr_t>(cd_raw) + 127) & ~uintptr_t(127));
  constexpr int KCH = KP / 8, NT = KP == 64 ? 4 : 8;
  const int tile = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
  const int s0 = p.row_start[seq] + rd.c0 * CD, s1 = min(p.row_start[seq + 1], s0 + rd.count * CD);
  if (s1 <= s0) return;
  const int H = p.heads, dk = p.dk, dv = p.dv, c0 = tile * DL_TILE;
  float* Sg = p.S + ((size_t)p.slots[seq] * H + h) * dk * dv;
  const size_t stride = (size_t)H * delta_record<KP>(dv);
  const uint8_t* rec = rd.scratch + ((size_t)seq * rd.count * H + h) * delta_record<KP>(dv);
  auto fetch = [&](uint8_t* dst, const uint8_t* src, int bytes) { for (int i = tid * 16; i < bytes; i += 256 * 16) cd_cp16(dst + i, src + i); };
  auto fetch_w = [&](const uint8_t* r) { fetch(sm.w[0], r, sizeof(sm.w)); };
  auto fetch_rest = [&](const uint8_t* r) { fetch(sm.q[0], r + sizeof(sm.w), sizeof(sm.q) + sizeof(sm.k) + sizeof(sm.p)); };
  // the warp's part of U and O: rows 16 (warp & 3), columns 32 (warp >> 2); of the state: rows 16 mt0, columns n0
  const int m0 = (warp & 3) * 16, o0 = (warp >> 2) * 32;
  const int mt0 = KP == 64 ? (warp & 3) : warp, n0 = KP == 64 ? (warp >> 2) * 32 : 0;
  float u[4][4], keep[2];
  auto fetch_u = [&](const uint8_t* r) {
    const float* src = reinterpret_cast<const float*>(r + sizeof(DeltaParts<KP>)) + (size_t)tile * CD * DL_TILE + (size_t)warp * 4 * 32 * 4;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) load4(src + (nt * 32 + lane) * 4, u[nt]);
    const float* kp = reinterpret_cast<const DeltaParts<KP>*>(r)->keep + mt0 * 16 + gq;
    keep[0] = kp[0]; keep[1] = kp[8];
  };
  fetch_w(rec);
  cd_commit();
  fetch_rest(rec);
  cd_commit();
  float st[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = mt0 * 16 + gq + 8 * e, col = c0 + n0 + nt * 8 + 2 * tq;
      float2 f = make_float2(0.f, 0.f);
      if (k < dk && col < dv) f = *reinterpret_cast<const float2*>(Sg + (size_t)k * dv + col);
      st[nt][2 * e] = f.x; st[nt][2 * e + 1] = f.y;
    }
  fetch_u(rec);
  const uint32_t aS0 = smem_u32(sm.s[0]), aS1 = smem_u32(sm.s[1]), aU0 = smem_u32(sm.u[0]), aU1 = smem_u32(sm.u[1]);
  for (int t0 = s0; t0 < s1; t0 += CD, rec += stride) {
    const int n = min(CD, s1 - t0);
    const bool more = t0 + CD < s1;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint32_t hi, lo;
        split2(st[nt][2 * e], st[nt][2 * e + 1], hi, lo);
        const uint32_t at = ms_off(mt0 * 16 + gq + 8 * e, (n0 >> 3) + nt, CDC) + 4 * tq;
        *reinterpret_cast<uint32_t*>(sm.s[0] + at) = hi;
        *reinterpret_cast<uint32_t*>(sm.s[1] + at) = lo;
      }
    cd_wait<1>();                                          // W is here
    __syncthreads();
    // ---- U = T diag(beta) V - W S
    product3<4>(u, smem_u32(sm.w[0]), smem_u32(sm.w[1]), KCH, m0, aS0, aS1, o0, KP / 16, lane);
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint32_t hi, lo;
        split2(u[nt][2 * e], u[nt][2 * e + 1], hi, lo);
        const uint32_t at = ms_off(m0 + gq + 8 * e, (o0 >> 3) + nt, CDC) + 4 * tq;
        *reinterpret_cast<uint32_t*>(sm.u[0] + at) = hi;
        *reinterpret_cast<uint32_t*>(sm.u[1] + at) = lo;
      }
    cd_wait<0>();                                          // the other tiles are here
    __syncthreads();
    const float k0 = keep[0], k1 = keep[1];
    if (more) { fetch_w(rec + stride); fetch_u(rec + stride); }
    cd_commit();
    // ---- O = (Q e^G) S + P U
    float o[4][4];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
    product3<4>(o, smem_u32(sm.q[0]), smem_u32(sm.q[1]), KCH, m0, aS0, aS1, o0, KP / 16, lane);
    product3<4>(o, smem_u32(sm.p[0]), smem_u32(sm.p[1]), CDC, m0, aU0, aU1, o0, (warp & 3) + 1, lane);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = m0 + gq + 8 * e;
      if (t < n) {
        float* orow = p.out + ((size_t)(t0 + t) * H + h) * dv;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          const int col = c0 + o0 + nt * 8 + 2 * tq;
          if (col < dv) *reinterpret_cast<float2*>(orow + col) = make_float2(o[nt][2 * e], o[nt][2 * e + 1]);
        }
      }
    }
    // ---- S <- e^{G_C} S + (K e^{G_C - G})^T U; A read transposed from the K tiles
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) { st[nt][0] *= k0; st[nt][1] *= k0; st[nt][2] *= k1; st[nt][3] *= k1; }
#pragma unroll 2
    for (int ks = 0; ks < CD / 16; ++ks) {
      uint32_t ah[4], al[4];
      const uint32_t ao = ms_off(ks * 16 + (lane & 7) + ((lane >> 4) << 3), mt0 * 2 + ((lane >> 3) & 1), KCH);
      ms_ldsm4t(smem_u32(sm.k[0]) + ao, ah[0], ah[1], ah[2], ah[3]);
      ms_ldsm4t(smem_u32(sm.k[1]) + ao, al[0], al[1], al[2], al[3]);
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
        const uint32_t bo = ms_off(ks * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), (n0 >> 3) + 2 * np + (lane >> 4), CDC);
        ms_ldsm4t(aU0 + bo, h0, h1, h2, h3);
        ms_ldsm4t(aU1 + bo, l0, l1, l2, l3);
        mma3(st[2 * np], ah, al, h0, h1, l0, l1);
        mma3(st[2 * np + 1], ah, al, h2, h3, l2, l3);
      }
    }
    __syncthreads();                                       // the tiles are no longer read
    if (more) fetch_rest(rec + stride);
    cd_commit();
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = mt0 * 16 + gq + 8 * e, col = c0 + n0 + nt * 8 + 2 * tq;
      if (k < dk && col < dv) *reinterpret_cast<float2*>(Sg + (size_t)k * dv + col) = make_float2(st[nt][2 * e], st[nt][2 * e + 1]);
    }
}

template <int KP>
static int delta_chunked_launch(const DeltaArgs<__nv_bfloat16>& p, int sequences, int chunks, int per_round, uint8_t* scratch, cudaStream_t s) {
  const int s1 = (int)sizeof(PartsSmem<KP>) + 128, s2 = (int)sizeof(ScanSmem<KP>) + 128;
  if (int r = opt_in_smem(delta_parts_kernel<KP>, s1)) return r;
  if (int r = opt_in_smem(delta_scan_kernel<KP>, s2)) return r;
  for (int c0 = 0; c0 < chunks; c0 += per_round) {
    const DeltaRound rd = {scratch, c0, chunks - c0 < per_round ? chunks - c0 : per_round};
    if (int r = launch_pdl(delta_parts_kernel<KP>, dim3(rd.count, p.heads, sequences), dim3(256), s1, s, 0, p, rd)) return r;
    if (int r = launch_pdl(delta_scan_kernel<KP>, dim3((p.dv + DL_TILE - 1) / DL_TILE, p.heads, sequences), dim3(256), s2, s, 0, p, rd)) return r;
  }
  return launch_result();
}

}  // namespace ff
using namespace ff;

// Bytes of scratch per (sequence, chunk of a round, head)
FF_EXPORT int ff_delta_chunk_record(int dk, int dv) { return (int)(dk <= 64 ? delta_record<64>(dv) : delta_record<128>(dv)); }

// As ff_delta_recurrent for BF16 rows, dk <= 128 and dk, dv multiples of 8. chunks: those of the longest sequence (64 rows each), taken
// per_round at a time; scratch: sequences * per_round * heads records, 16-byte aligned.
FF_EXPORT int ff_delta_chunked(const void* x, const float* unit, const float* decay, const void* beta, const float* rate, const float* dt_bias,
                               float* S, float* out, const int* row_start, const int* slots, int sequences, int ldx, int ldd, int ldb, int heads,
                               int kv_heads, int dk, int dv, int chunks, int per_round, void* scratch, cudaStream_t s) {
  if (sequences <= 0 || sequences > 65535 || heads <= 0 || heads > 65535 || kv_heads <= 0 || heads % kv_heads || dk <= 0 || dk % 8 || dv <= 0 || dv % 8)
    return FF_HOST_BAD_SHAPE;
  if (ldx < 2 * kv_heads * dk + heads * dv || ldd < heads * dk || ldb < heads || chunks < 1 || per_round < 1 || scratch == nullptr) return FF_HOST_BAD_SHAPE;
  if (dk > 128) return FF_HOST_TOO_LARGE;
  if (ldx % 8 || ldd % 4 || (reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(S) & 15) || (reinterpret_cast<uintptr_t>(out) & 15) ||
      (reinterpret_cast<uintptr_t>(decay) & 15) || (reinterpret_cast<uintptr_t>(dt_bias) & 15) || (reinterpret_cast<uintptr_t>(scratch) & 15)) return FF_HOST_BAD_ALIGN;
  const DeltaArgs<__nv_bfloat16> p = {(const __nv_bfloat16*)x, unit, decay, (const __nv_bfloat16*)beta, rate, dt_bias, S, out, row_start, slots, ldx, ldd, ldb, heads, kv_heads, dk, dv};
  if (dk <= 64) return delta_chunked_launch<64>(p, sequences, chunks, per_round, (uint8_t*)scratch, s);
  return delta_chunked_launch<128>(p, sequences, chunks, per_round, (uint8_t*)scratch, s);
}
