// Matrix-valued states with scalar gates: the matrix memory of xLSTM (mLSTM) and, below it, the state space of Mamba-2.
// Matrix memory with exponential gates. Per head, with log gates i_t = cap tanh(z_i / cap) and
// f_t = logsigmoid(cap tanh(z_f / cap)) and a running maximum m (from 0):
//   m_t = max(f_t + m_{t-1}, i_t)
//   S_t = e^{f_t + m_{t-1} - m_t} S_{t-1} + e^{i_t - m_t} k_t v_t^T          n_t likewise with k_t alone
//   o_t = S_t^T q_t / (max(|n_t . q_t|, e^{-m_t}) + 1e-6)
// Three forms over packed projection rows [q | k | v | gate] of several sequences, the state addressed by slot:
//   recurrent : token by token, FP32 arithmetic, BF16 or FP32 rows (decode; 32-bit prompts). The state of 64 value columns
//               sits in registers while the tokens of a sequence pass.
//   chunked   : prompts, BF16 rows, 64 tokens at a time. With F_t = f_1 + .. + f_t over the chunk, a_j = i_j - F_j and
//               M_t = max(m_0, max_{j<=t} a_j) every exponent below is at most zero:
//                 O = e^{m_0 - M_t} Q S_0 + P V,   P[t,j] = e^{a_j - M_t} (q_t . k_j)  (j <= t)
//                 S <- e^{m_0 - M_C} S_0 + K^T (e^{a_j - M_C} V),   m <- F_C + M_C
//               four mma.sync products per chunk; S in FP32 accumulator registers, its operand copy, P and the weighted V
//               split into a BF16 value and a BF16 remainder so that nothing of the recurrence is cut to 8 bits.
//   segmented : a long prompt with few heads: the chunked form runs over segments of the prompt side by side. First every
//               segment's own contribution to the state (from zero), then a scan over the segments, then the outputs from
//               each segment's starting state.
// out : heads divided by their root mean square, times a weight and the sigmoid of the gate columns.
// State space (SSD): per head, with steps d_t = softplus(z_t + bias), a = -exp(A_log) and input and output maps B, C shared by the heads
// of a group,
//   S_t = e^{a d_t} S_{t-1} + d_t B_t x_t^T        y_t = S_t^T C_t + D x_t
// It is the recurrence above with q = C, k = B, v = x, f_t = a d_t, i_t = ln d_t, no normaliser and no running maximum (weights are
// e^{F_t - F_j} d_j as they are: M_t = -F_t in the chunked form), and runs in the same kernels (SSD = true).
// ssd_out : y silu(z), divided by the root mean square of its part of the row, times a weight.
// A CTA owns 64 value columns ("tile") and keeps a copy of n and m of its own, so no two CTAs share state.
#include "dtype_io.cuh"
#include "host_util.h"
#include "mma_sync.cuh"

namespace ff {

constexpr int ML_TILE = 64;

struct LogGates { float i, f; };
struct Step { float d, f; };          // step size and logarithm of the decay
__device__ __forceinline__ Step ssd_step(float z, float a) {
  const float d = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
  return {d, a * d};
}
__device__ __forceinline__ LogGates log_gates(float zi, float zf, float cap) {
  const float f = cap * tanhf(zf / cap);
  return {cap * tanhf(zi / cap), fminf(f, 0.f) - log1pf(expf(-fabsf(f)))};
}

// what every form gets
template <typename T>
struct MlstmArgs {
  const T* x;                        // packed rows: q at h * dk, k at (H + h) * dk, v at 2 H dk + h * dv
  const float* gates;                // [rows, ldg]: z_i of the heads, then z_f
  const float* gate_bias;            // [2 H]
  float* S; float* n; float* m;      // [slots, H, dk, dv], [slots, H, tiles, dk], [slots, H, tiles]
  float* out;                        // [rows, H, dv]
  const int* row_start; const int* slots;
  int ldx, ldg, heads, dk, dv, tiles;
  float qscale, cap;
  int kheads;                        // heads of q and k (SSD: groups; q at g * dk, k at (kheads + g) * dk, v at 2 kheads dk + h * dv)
  // SSD: step logits [rows, ldg] in the rows' type (gates unused), their bias in gate_bias [H], a and D per head
  const T* steps; const float* a; const float* skip;
};

// ---------------------------------------------------------------------------------------
// recurrent: grid (tiles, heads, sequences), 256 threads = 16 float4 columns x 16 key groups; R key rows per thread
// ---------------------------------------------------------------------------------------
template <typename T, int R, bool SSD>
__global__ void __launch_bounds__(256)
mlstm_recurrent_kernel(const MlstmArgs<T> p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float sq[16 * R], sk[16 * R];
  __shared__ __align__(16) float s_o[2][8][ML_TILE];
  __shared__ float s_nq[2][8];
  const int tile = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r0 = p.row_start[seq], r1 = p.row_start[seq + 1];
  if (r1 <= r0) return;
  const int H = p.heads, dk = p.dk, dv = p.dv, slot = p.slots[seq];
  const int c = tid & 15, kg = tid >> 4, col = tile * ML_TILE + c * 4;
  const bool live = col < dv;
  float* Sg = p.S + ((size_t)slot * H + h) * dk * dv + col;
  const size_t ntile = ((size_t)slot * H + h) * p.tiles + tile;
  const int KH = p.kheads, kh = SSD ? h / (H / KH) : h;
  float* ng = SSD ? nullptr : p.n + ntile * dk;
  float st[R][4];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int k = kg + 16 * r;
    if (live && k < dk) load4(Sg + (size_t)k * dv, st[r]);
    else st[r][0] = st[r][1] = st[r][2] = st[r][3] = 0.f;
  }
  constexpr int NN = (16 * R + 255) / 256;                 // elements of n a thread owns
  float nv[NN];
#pragma unroll
  for (int j = 0; j < NN; ++j) nv[j] = !SSD && tid + 256 * j < dk ? ng[tid + 256 * j] : 0.f;
  float m = SSD ? 0.f : p.m[ntile];
  const float bi = p.gate_bias[h], bf = SSD ? p.a[h] : p.gate_bias[H + h], skip = SSD ? p.skip[h] : 0.f;
  for (int row = r0; row < r1; ++row) {
    const int par = (row - r0) & 1;
    const T* xr = p.x + (size_t)row * p.ldx;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (live) load4(xr + (size_t)2 * KH * dk + (size_t)h * dv + col, v);
    float keep, add;
    if constexpr (SSD) {
      const Step g = ssd_step(to_float(p.steps[(size_t)row * p.ldg + h]) + bi, bf);
      keep = expf(g.f);
      add = g.d;
    } else {
      const LogGates g = log_gates(p.gates[(size_t)row * p.ldg + h] + bi, p.gates[(size_t)row * p.ldg + H + h] + bf, p.cap);
      const float mn = fmaxf(g.f + m, g.i);
      keep = expf(g.f + m - mn);
      add = expf(g.i - mn);
      m = mn;
    }
    float nq = 0.f;
#pragma unroll
    for (int j = 0; j < NN; ++j) {
      const int k = tid + 256 * j;
      if (k < dk) {
        const float qk = to_float(xr[(size_t)kh * dk + k]) * p.qscale, kk = to_float(xr[(size_t)(KH + kh) * dk + k]);
        sq[k] = qk; sk[k] = kk;
        if (!SSD) {
          nv[j] = keep * nv[j] + add * kk;
          nq = fmaf(nv[j], qk, nq);
        }
      } else if (k < 16 * R) { sq[k] = 0.f; sk[k] = 0.f; }
    }
    nq = warp_sum(nq);
    if (lane == 0) s_nq[par][warp] = nq;
    __syncthreads();
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const float kk = add * sk[kg + 16 * r], qk = sq[kg + 16 * r];
#pragma unroll
      for (int j = 0; j < 4; ++j) { st[r][j] = fmaf(kk, v[j], keep * st[r][j]); acc[j] = fmaf(qk, st[r][j], acc[j]); }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], 16);
    if (lane < 16) store4(&s_o[par][warp][c * 4], acc);
    __syncthreads();
    if (tid < ML_TILE && tile * ML_TILE + tid < dv) {
      float o = 0.f, d = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) { o += s_o[par][w][tid]; d += s_nq[par][w]; }
      if (SSD) o = fmaf(skip, to_float(xr[(size_t)2 * KH * dk + (size_t)h * dv + tile * ML_TILE + tid]), o);
      p.out[((size_t)row * H + h) * dv + tile * ML_TILE + tid] = SSD ? o : o / (fmaxf(fabsf(d), expf(-m)) + 1e-6f);
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int k = kg + 16 * r;
    if (live && k < dk) store4(Sg + (size_t)k * dv, st[r]);
  }
  if (SSD) return;
#pragma unroll
  for (int j = 0; j < NN; ++j) if (tid + 256 * j < dk) ng[tid + 256 * j] = nv[j];
  if (tid == 0) p.m[ntile] = m;
}

// ---------------------------------------------------------------------------------------
// chunked: grid (tiles, heads, sequences x segments), 256 threads. KP: key width padded to 64, 128 or 256.
// ---------------------------------------------------------------------------------------
constexpr int MC = 64;               // tokens per chunk
constexpr int MGB = 4;               // chunks whose gates are worked out together, a warp each
constexpr int MTC = ML_TILE / 8;     // 16-byte chunks per row of a 64-column tile

template <int KP>
struct MlstmSmem {
  uint8_t q[MC * KP * 2], k[MC * KP * 2], v[MC * ML_TILE * 2];
  uint8_t s[2][KP * ML_TILE * 2];    // operand copy of the state: value, remainder
  uint8_t vw[2][MC * ML_TILE * 2];   // e^{a_j - M_C} v_j: value, remainder
  uint8_t p[2][MC * MC * 2];         // P: value, remainder
  float n[KP], np[4][KP];            // n as the chunk finds it; its next value in four parts (16 tokens each)
  float ga[MGB][MC], gf[MGB][MC], gm[MGB][MC];             // a_j, F_j and max_{i<=j} a_i of the next chunks
  float top[MC], carry[MC], floor[MC];                     // M_t, e^{m_0 - M_t}, e^{-m_t}
  alignas(16) float kw[MC];                                // e^{a_j - M_C}
  float qn[MC], rs[2][MC];
};

// Segments of a long prompt. count == 1: a sequence is one segment, the state comes from and goes to its slot.
// pass 1: the segment's own contribution (S from zero, m from minus infinity), no output, not needed of the last segment;
// pass 2: outputs from the starting state in S / n / m_start, the last segment writes the slot.
struct MlstmSegments {
  int count, len, pass;
  float* S; float* n;                // [sequence, segment, H, dk, dv], [.., H, tiles, dk]
  float* m_own; float* f_own; float* m_start;   // [sequence, segment, H, tiles]
};

__device__ __forceinline__ void store_split(uint8_t (*tile)[MC * ML_TILE * 2], int row, int col, float x, float y) {
  const float xh = __bfloat162float(__float2bfloat16(x)), yh = __bfloat162float(__float2bfloat16(y));
  ms_store2(tile[0], row, col, MTC, xh, yh);
  ms_store2(tile[1], row, col, MTC, x - xh, y - yh);
}

template <int KP, bool SSD>
__global__ void __launch_bounds__(256, KP == 256 ? 1 : 2)
mlstm_chunk_kernel(const MlstmArgs<__nv_bfloat16> p, const MlstmSegments sg) {
  pdl_trigger();
  pdl_wait();
  constexpr int KCH = KP / 8;
  constexpr int MT = KP == 256 ? 2 : 1;                    // 16-row tiles of the state per warp
  constexpr int NT = KP == 64 ? 4 : 8;                     // 8-column tiles of the state per warp
  extern __shared__ __align__(128) uint8_t ml_raw[];
  MlstmSmem<KP>& sm = *reinterpret_cast<MlstmSmem<KP>*>((reinterpret_cast<uintptr_t>(ml_raw) + 127) & ~uintptr_t(127));
  const int tile = blockIdx.x, h = blockIdx.y, seq = blockIdx.z / sg.count, seg = blockIdx.z % sg.count;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
  const int s0 = p.row_start[seq], s1 = p.row_start[seq + 1];
  const int r0 = s0 + seg * sg.len, r1 = sg.count == 1 ? s1 : min(s1, r0 + sg.len);
  if (r1 <= r0) return;
  const bool last = r1 == s1, own = sg.pass == 1;
  if (own && last) return;
  const int H = p.heads, dk = p.dk, dv = p.dv, slot = p.slots[seq], c0 = tile * ML_TILE;
  const size_t hs = (size_t)slot * H + h, hseg = (size_t)blockIdx.z * H + h;
  const int KH = p.kheads, kh = SSD ? h / (H / KH) : h;
  const float* Sin = sg.count == 1 ? p.S + hs * dk * dv : sg.S + hseg * dk * dv;
  const float* nin = SSD ? nullptr : (sg.count == 1 ? p.n + (hs * p.tiles + tile) * dk : sg.n + (hseg * p.tiles + tile) * dk);
  const uint32_t aQ = smem_u32(sm.q), aK = smem_u32(sm.k), aV = smem_u32(sm.v);

  // state fragments: rows (key elements) of tile mt0 + i, columns n0 .. n0 + 8 NT
  const int mt0 = KP == 64 ? (warp & 3) : warp * MT, n0 = KP == 64 ? (warp >> 2) * 32 : 0;
  float st[MT][NT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int k = (mt0 + i) * 16 + gq + 8 * e, col = c0 + n0 + nt * 8 + 2 * tq;
        float2 f = make_float2(0.f, 0.f);
        if (!own && k < dk && col < dv) f = *reinterpret_cast<const float2*>(Sin + (size_t)k * dv + col);
        st[i][nt][2 * e] = f.x; st[i][nt][2 * e + 1] = f.y;
      }
  if (!SSD) for (int k = tid; k < KP; k += 256) {
    sm.np[0][k] = !own && k < dk ? nin[k] : 0.f;
    sm.np[1][k] = sm.np[2][k] = sm.np[3][k] = 0.f;
  }
  float m = SSD ? 0.f : (own ? -INFINITY : (sg.count == 1 ? p.m[hs * p.tiles + tile] : sg.m_start[hseg * p.tiles + tile]));
  float f_all = 0.f;
  const float bi = p.gate_bias[h], bf = SSD ? p.a[h] : p.gate_bias[H + h], skip = SSD ? p.skip[h] : 0.f;
  auto gates_of = [&](int row) -> LogGates {
    if constexpr (SSD) {
      const Step g = ssd_step(to_float(p.steps[(size_t)row * p.ldg + h]) + bi, bf);
      return {logf(g.d), g.f};
    } else {
      const float* z = p.gates + (size_t)row * p.ldg;
      return log_gates(z[h] + bi, z[H + h] + bf, p.cap);
    }
  };

  for (int t0 = r0, ci = 0; t0 < r1; t0 += MC, ci = (ci + 1) % MGB) {
    const int n = min(MC, r1 - t0);
    __syncthreads();                                       // the previous chunk's tiles are no longer read
    if (ci == 0) {
      // gates, prefix sums of f and prefix maxima of a of the next chunks, two tokens per lane; past the end: f = 0, a = -inf
      const int ta = 2 * lane, tb = ta + 1, tw = t0 + warp * MC;
      if (warp < MGB && tw < r1) {
        LogGates g0 = {-INFINITY, 0.f}, g1 = g0;
        if (tw + ta < r1) g0 = gates_of(tw + ta);
        if (tw + tb < r1) g1 = gates_of(tw + tb);
        float run = g0.f + g1.f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const float up = __shfl_up_sync(0xffffffffu, run, o); if (lane >= o) run += up; }
        const float f1 = run, f0 = run - g1.f, a0 = g0.i - f0, a1 = g1.i - f1;
        float mx = fmaxf(a0, a1);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const float up = __shfl_up_sync(0xffffffffu, mx, o); if (lane >= o) mx = fmaxf(mx, up); }
        float before = __shfl_up_sync(0xffffffffu, mx, 1);
        if (lane == 0) before = -INFINITY;
        sm.ga[warp][ta] = a0; sm.ga[warp][tb] = a1;
        sm.gf[warp][ta] = f0; sm.gf[warp][tb] = f1;
        sm.gm[warp][ta] = fmaxf(before, a0); sm.gm[warp][tb] = mx;
      }
      __syncthreads();
    }
    const float Fc = sm.gf[ci][MC - 1], Mc = SSD ? -Fc : fmaxf(m, sm.gm[ci][MC - 1]), keep = expf(m - Mc);
    if (tid < MC) {
      const float M = SSD ? -sm.gf[ci][tid] : fmaxf(m, sm.gm[ci][tid]);
      sm.top[tid] = M;
      sm.carry[tid] = expf(m - M);
      sm.floor[tid] = expf(-(sm.gf[ci][tid] + M));
      sm.kw[tid] = expf(sm.ga[ci][tid] - Mc);
    }
    if (!SSD) for (int k = tid; k < KP; k += 256) sm.n[k] = (sm.np[0][k] + sm.np[1][k]) + (sm.np[2][k] + sm.np[3][k]);
    // ---- tiles of the chunk; rows past n and columns past the heads are zero
    for (int i = tid; i < MC * KCH; i += 256) {
      const int t = i / KCH, cch = i - t * KCH;
      uint4 qv = make_uint4(0, 0, 0, 0), kv = qv;
      if (t < n && cch * 8 < dk) {
        const __nv_bfloat16* xr = p.x + (size_t)(t0 + t) * p.ldx + cch * 8;
        if (!own) qv = *reinterpret_cast<const uint4*>(xr + (size_t)kh * dk);
        kv = *reinterpret_cast<const uint4*>(xr + (size_t)(KH + kh) * dk);
      }
      if (!own) *reinterpret_cast<uint4*>(sm.q + ms_off(t, cch, KCH)) = qv;
      *reinterpret_cast<uint4*>(sm.k + ms_off(t, cch, KCH)) = kv;
    }
    for (int i = tid; i < MC * MTC; i += 256) {
      const int t = i / MTC, cch = i - t * MTC;
      uint4 vv = make_uint4(0, 0, 0, 0);
      if (t < n && c0 + cch * 8 < dv)
        vv = *reinterpret_cast<const uint4*>(p.x + (size_t)(t0 + t) * p.ldx + (size_t)2 * KH * dk + (size_t)h * dv + c0 + cch * 8);
      *reinterpret_cast<uint4*>(sm.v + ms_off(t, cch, MTC)) = vv;
    }
    // the next chunk's rows on their way into the L2 cache
    for (int i = tid; i < MC * (2 * KP / 64 + 1); i += 256) {
      const int t = t0 + MC + i % MC, part = i / MC;
      if (t >= r1) continue;
      const __nv_bfloat16* xr = p.x + (size_t)t * p.ldx;
      const int col = part * 64 - (part >= KP / 64 ? KP : 0);
      const __nv_bfloat16* at = part == 2 * KP / 64 ? xr + (size_t)2 * KH * dk + (size_t)h * dv + c0 : xr + (size_t)(part >= KP / 64 ? KH + kh : kh) * dk + col;
      if (part == 2 * KP / 64 || col < dk) asm volatile("prefetch.global.L2 [%0];" ::"l"(at));
    }
    if (!own) {
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int k = (mt0 + i) * 16 + gq + 8 * e, col = n0 + nt * 8 + 2 * tq;
            const float x = st[i][nt][2 * e], y = st[i][nt][2 * e + 1];
            const float xh = __bfloat162float(__float2bfloat16(x)), yh = __bfloat162float(__float2bfloat16(y));
            ms_store2(sm.s[0], k, col, MTC, xh, yh);
            ms_store2(sm.s[1], k, col, MTC, x - xh, y - yh);
          }
    }
    __syncthreads();

    // ---- weighted values
    for (int i = tid; i < MC * ML_TILE / 2; i += 256) {
      const int t = i / (ML_TILE / 2), col = (i - t * (ML_TILE / 2)) * 2;
      const float2 f = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm.v + ms_off(t, col >> 3, MTC) + (col & 7) * 2));
      const float w = sm.kw[t];
      store_split(sm.vw, t, col, f.x * w, f.y * w);
    }
    if (!own) {
      // ---- P = e^{a_j - M_t} (q . k) qscale, row sums
      const int m0 = (warp & 3) * 16, half = warp >> 2;
      float qk[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) qk[i][0] = qk[i][1] = qk[i][2] = qk[i][3] = 0.f;
      ms_product<4, KP / 16, false>(qk, aQ, KCH, m0, aK, KCH, half * 32, lane);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = m0 + gq + 8 * e;
        const float top = sm.top[t];
        float sum = 0.f;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          float v[2];
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int i = half * 32 + nt * 8 + 2 * tq + j;
            v[j] = i <= t ? __expf(sm.ga[ci][i] - top) * p.qscale * qk[nt][2 * e + j] : 0.f;
            sum += v[j];
          }
          store_split(sm.p, t, half * 32 + nt * 8 + 2 * tq, v[0], v[1]);
        }
        if (!SSD) {
          sum += __shfl_xor_sync(0xffffffffu, sum, 1);
          sum += __shfl_xor_sync(0xffffffffu, sum, 2);
          if (tq == 0) sm.rs[half][t] = sum;
        }
      }
      // ---- q . n of the incoming state: four threads per token
      if (!SSD) {
        const int t = tid >> 2, part = tid & 3;
        float d = 0.f;
        for (int cch = part; cch < KCH; cch += 4) {
          const uint4 u = *reinterpret_cast<const uint4*>(sm.q + ms_off(t, cch, KCH));
          const uint32_t* w = reinterpret_cast<const uint32_t*>(&u);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float2 f = unpack_bf16x2(w[j]);
            d = fmaf(f.x, sm.n[cch * 8 + 2 * j], d);
            d = fmaf(f.y, sm.n[cch * 8 + 2 * j + 1], d);
          }
        }
        d += __shfl_xor_sync(0xffffffffu, d, 1);
        d += __shfl_xor_sync(0xffffffffu, d, 2);
        if (part == 0) sm.qn[t] = d * p.qscale;
      }
    }
    __syncthreads();

    if (!own) {
      // ---- O = (carry Q S_0 + P V) / den
      const int m0 = (warp & 3) * 16, o0 = (warp >> 2) * 32;
      float oa[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) oa[i][0] = oa[i][1] = oa[i][2] = oa[i][3] = 0.f;
      ms_product<4, KP / 16, true>(oa, aQ, KCH, m0, smem_u32(sm.s[0]), MTC, o0, lane);
      ms_product<4, KP / 16, true>(oa, aQ, KCH, m0, smem_u32(sm.s[1]), MTC, o0, lane);
      const float ca = sm.carry[m0 + gq] * p.qscale, cb = sm.carry[m0 + gq + 8] * p.qscale;
#pragma unroll
      for (int i = 0; i < 4; ++i) { oa[i][0] *= ca; oa[i][1] *= ca; oa[i][2] *= cb; oa[i][3] *= cb; }
      ms_product<4, MC / 16, true>(oa, smem_u32(sm.p[0]), MTC, m0, aV, MTC, o0, lane);
      ms_product<4, MC / 16, true>(oa, smem_u32(sm.p[1]), MTC, m0, aV, MTC, o0, lane);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = m0 + gq + 8 * e;
        if (t < n) {
          float inv = 1.0f;
          if (!SSD) {
            const float d = sm.qn[t] * sm.carry[t] + sm.rs[0][t] + sm.rs[1][t];
            inv = 1.0f / (fmaxf(fabsf(d), sm.floor[t]) + 1e-6f);
          }
          float* orow = p.out + ((size_t)(t0 + t) * H + h) * dv;
#pragma unroll
          for (int nt = 0; nt < 4; ++nt) {
            const int col = c0 + o0 + nt * 8 + 2 * tq;
            float2 o = make_float2(oa[nt][2 * e] * inv, oa[nt][2 * e + 1] * inv);
            if (SSD) {
              const int lc = col - c0;
              const float2 x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm.v + ms_off(t, lc >> 3, MTC) + (lc & 7) * 2));
              o.x = fmaf(skip, x.x, o.x); o.y = fmaf(skip, x.y, o.y);
            }
            if (col < dv) *reinterpret_cast<float2*>(orow + col) = o;
          }
        }
      }
    }
    // ---- S <- keep S + K^T (weighted V); A read transposed from the K tile
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) { st[i][nt][0] *= keep; st[i][nt][1] *= keep; st[i][nt][2] *= keep; st[i][nt][3] *= keep; }
#pragma unroll
    for (int ks = 0; ks < MC / 16; ++ks) {
      uint32_t a[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i)
        ms_ldsm4t(aK + ms_off(ks * 16 + (lane & 7) + ((lane >> 4) << 3), (mt0 + i) * 2 + ((lane >> 3) & 1), KCH), a[i][0], a[i][1], a[i][2], a[i][3]);
#pragma unroll
      for (int w = 0; w < 2; ++w)
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          uint32_t b0, b1, b2, b3;
          const int krow = ks * 16 + (((lane >> 3) & 1) << 3) + (lane & 7);
          ms_ldsm4t(smem_u32(sm.vw[w]) + ms_off(krow, (n0 >> 3) + 2 * np + (lane >> 4), MTC), b0, b1, b2, b3);
#pragma unroll
          for (int i = 0; i < MT; ++i) { ms_mma(st[i][2 * np], a[i], b0, b1); ms_mma(st[i][2 * np + 1], a[i], b2, b3); }
        }
    }
    // ---- n <- keep n + sum_j e^{a_j - M_C} k_j: a thread takes two key elements and 16 tokens
    if (!SSD) for (int i = tid; i < 2 * KP; i += 256) {
      const int k = (i % (KP / 2)) * 2, part = i / (KP / 2);
      float x = part == 0 ? keep * sm.n[k] : 0.f, y = part == 0 ? keep * sm.n[k + 1] : 0.f;
#pragma unroll
      for (int t = 0; t < 16; ++t) {
        const float w = sm.kw[part * 16 + t];
        const float2 f = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm.k + ms_off(part * 16 + t, k >> 3, KCH) + (k & 7) * 2));
        x = fmaf(w, f.x, x);
        y = fmaf(w, f.y, y);
      }
      sm.np[part][k] = x; sm.np[part][k + 1] = y;
    }
    if (!SSD) m = Fc + Mc;
    f_all += Fc;
  }
  __syncthreads();
  // ---- state out
  if (!own && !last) return;
  float* So = own ? sg.S + hseg * dk * dv : p.S + hs * dk * dv;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int k = (mt0 + i) * 16 + gq + 8 * e, col = c0 + n0 + nt * 8 + 2 * tq;
        if (k < dk && col < dv) *reinterpret_cast<float2*>(So + (size_t)k * dv + col) = make_float2(st[i][nt][2 * e], st[i][nt][2 * e + 1]);
      }
  if (SSD) {
    if (own && tid == 0) sg.f_own[hseg * p.tiles + tile] = f_all;
    return;
  }
  float* no = own ? sg.n + (hseg * p.tiles + tile) * dk : p.n + (hs * p.tiles + tile) * dk;
  for (int k = tid; k < dk; k += 256) no[k] = (sm.np[0][k] + sm.np[1][k]) + (sm.np[2][k] + sm.np[3][k]);
  if (tid == 0) {
    if (own) { sg.m_own[hseg * p.tiles + tile] = m; sg.f_own[hseg * p.tiles + tile] = f_all; }
    else p.m[hs * p.tiles + tile] = m;
  }
}

// Starting state of every segment from the slot's state and the segments' own contributions, in place.
// grid (blocks over dk * dv / 4 and n, heads, sequences), 256 threads
template <bool SSD>
__global__ void __launch_bounds__(256)
mlstm_scan_kernel(const MlstmArgs<__nv_bfloat16> p, const MlstmSegments sg, int s_blocks) {
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, seq = blockIdx.z, H = p.heads;
  const int rows = p.row_start[seq + 1] - p.row_start[seq];
  const int segs = (rows + sg.len - 1) / sg.len;
  if (segs <= 0) return;
  const size_t hs = (size_t)p.slots[seq] * H + h;
  const bool is_n = blockIdx.x >= s_blocks;
  const int per = is_n ? p.tiles * p.dk : p.dk * p.dv;     // multiples of 16
  const int i = ((is_n ? blockIdx.x - s_blocks : blockIdx.x) * 256 + threadIdx.x) * 4;
  const bool live = i < per;
  float cur[4] = {0.f, 0.f, 0.f, 0.f};
  if (live) load4((is_n ? p.n + hs * p.tiles * p.dk : p.S + hs * p.dk * p.dv) + i, cur);
  float m = SSD ? 0.f : p.m[hs * p.tiles];                 // the tiles' copies of m are equal
  for (int s = 0; s < segs; ++s) {
    const size_t hseg = ((size_t)seq * sg.count + s) * H + h;
    float* at = (is_n ? sg.n + hseg * p.tiles * p.dk : sg.S + hseg * p.dk * p.dv) + i;
    float own[4] = {0.f, 0.f, 0.f, 0.f};
    const bool more = s + 1 < segs;
    if (live && more) load4(at, own);
    if (live) store4(at, cur);
    if (!SSD && blockIdx.x == 0 && threadIdx.x < p.tiles) sg.m_start[hseg * p.tiles + threadIdx.x] = m;
    if (!more) break;
    const float mo = SSD ? 0.f : sg.m_own[hseg * p.tiles], fo = sg.f_own[hseg * p.tiles];
    const float mn = SSD ? 0.f : fmaxf(fo + m, mo), keep = expf(fo + m - mn), add = expf(mo - mn);
#pragma unroll
    for (int j = 0; j < 4; ++j) cur[j] = keep * cur[j] + add * own[j];
    m = mn;
  }
}

// ---------------------------------------------------------------------------------------
// out: one warp per (row, head): y = o / rms(o) * w * sigmoid(gate); dv true elements `vdim`, padded to dv
// ---------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
mlstm_out_kernel(const float* __restrict__ o, const T* __restrict__ gate, int ldg, const float* __restrict__ w, T* __restrict__ y, int rows,
                 int heads, int vdim, int dv, float eps) {
  pdl_trigger();
  pdl_wait();
  const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= (long long)rows * heads) return;
  const int row = (int)(item / heads), h = (int)(item % heads);
  const float* src = o + item * dv;
  float ss = 0.f;
  for (int c = lane * 4; c < dv; c += 128) {
    float v[4];
    load4(src + c, v);
#pragma unroll
    for (int j = 0; j < 4; ++j) ss = fmaf(v[j], v[j], ss);   // the padding of a head is zero
  }
  const float r = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
  for (int c = lane * 4; c < dv; c += 128) {
    float v[4], g[4], f[4];
    load4(src + c, v);
    load4(gate + (size_t)row * ldg + (size_t)h * dv + c, g);
    load4(w + (size_t)h * dv + c, f);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = v[j] * r * f[j] * sigmoid_f(g[j]);
    store4(y + item * dv + c, v);
  }
}

// ssd_out: a block per (row, part of the row): y = o silu(z), divided by the part's root mean square, times w. Heads stand dv apart, of
// which the first vdim elements count; the parts are equal pieces of the heads' own elements put together.
template <typename T>
__global__ void __launch_bounds__(256)
ssd_out_kernel(const float* __restrict__ o, const T* __restrict__ z, int ldz, const float* __restrict__ w, T* __restrict__ y, int heads, int vdim,
               int dv, int part, float eps) {
  pdl_trigger();
  extern __shared__ __align__(16) float so_v[];            // [part]
  __shared__ float s_red[8];
  pdl_wait();
  const int row = blockIdx.y, tid = threadIdx.x, first = blockIdx.x * part;
  const size_t base = (size_t)row * heads * dv;
  float ss = 0.f;
  const bool vec = vdim == dv && part % 4 == 0;
  if (vec) {
    for (int c = tid * 4; c < part; c += blockDim.x * 4) {
      float a[4], g[4];
      load4(o + base + first + c, a);
      load4(z + (size_t)row * ldz + first + c, g);
#pragma unroll
      for (int j = 0; j < 4; ++j) { a[j] *= g[j] * sigmoid_f(g[j]); ss = fmaf(a[j], a[j], ss); }
      store4(so_v + c, a);
    }
  } else {
    for (int c = tid; c < part; c += blockDim.x) {
      const int h = (first + c) / vdim, at = h * dv + (first + c) - h * vdim;
      const float g = to_float(z[(size_t)row * ldz + at]), a = o[base + at] * g * sigmoid_f(g);
      ss = fmaf(a, a, ss);
      so_v[c] = a;
    }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) s_red[tid >> 5] = ss;
  __syncthreads();
  const float r = 1.0f / sqrtf(warp_sum((tid & 31) < (int)(blockDim.x >> 5) ? s_red[tid & 31] : 0.f) / (float)part + eps);
  if (vec) {
    for (int c = tid * 4; c < part; c += blockDim.x * 4) { // the thread's own elements again
      float a[4], f[4];
      load4(so_v + c, a);
      load4(w + first + c, f);
#pragma unroll
      for (int j = 0; j < 4; ++j) a[j] *= r * f[j];
      store4(y + base + first + c, a);
    }
    return;
  }
  for (int c = tid; c < part; c += blockDim.x) {
    const int h = (first + c) / vdim, e = (first + c) - h * vdim, at = h * dv + e;
    from_float(y + base + at, so_v[c] * r * w[at]);
    if (e == vdim - 1)
      for (int k = vdim; k < dv; ++k) from_float(y + base + h * dv + k, 0.f);
  }
}

template <bool SSD, typename T>
static int mlstm_check(const MlstmArgs<T>& p, int sequences) {
  if (sequences <= 0 || sequences > 65535 || p.heads <= 0 || p.heads > 65535 || p.dk <= 0 || p.dk % 16 || p.dv <= 0 || p.dv % 16) return FF_HOST_BAD_SHAPE;
  if (p.tiles != (p.dv + ML_TILE - 1) / ML_TILE || p.kheads <= 0 || p.heads % p.kheads) return FF_HOST_BAD_SHAPE;
  if (SSD ? p.ldg < p.heads : (!(p.cap > 0.f) || p.ldg < 2 * p.heads || p.kheads != p.heads)) return FF_HOST_BAD_SHAPE;
  if (p.ldx % 8 || (reinterpret_cast<uintptr_t>(p.x) & 15) || (reinterpret_cast<uintptr_t>(p.S) & 15)) return FF_HOST_BAD_ALIGN;
  return FF_HOST_OK;
}

template <bool SSD, typename T>
static int mlstm_recurrent_launch(const MlstmArgs<T>& p, int sequences, cudaStream_t s) {
  if (int r = mlstm_check<SSD>(p, sequences)) return r;
  auto go = [&](auto kern) -> int {
    if (int r = launch_pdl(kern, dim3(p.tiles, p.heads, sequences), dim3(256), 0, s, 0, p)) return r;
    return launch_result();
  };
  if (p.dk <= 16) return go(mlstm_recurrent_kernel<T, 1, SSD>);
  if (p.dk <= 32) return go(mlstm_recurrent_kernel<T, 2, SSD>);
  if (p.dk <= 64) return go(mlstm_recurrent_kernel<T, 4, SSD>);
  if (p.dk <= 128) return go(mlstm_recurrent_kernel<T, 8, SSD>);
  if (p.dk <= 256) return go(mlstm_recurrent_kernel<T, 16, SSD>);
  if (p.dk <= 512) return go(mlstm_recurrent_kernel<T, 32, SSD>);
  return FF_HOST_TOO_LARGE;
}

// segments > 1: every sequence in up to `segments` pieces of seg_len rows; scratch holds sequences * segments * heads *
// (dk * dv + tiles * (dk + 3)) floats
template <bool SSD>
static int mlstm_chunked_launch(const MlstmArgs<__nv_bfloat16>& p, int sequences, int segments, int seg_len, float* scratch, cudaStream_t s) {
  if (int r = mlstm_check<SSD>(p, sequences)) return r;
  if (segments < 1 || (long long)sequences * segments > 65535 || (segments > 1 && (seg_len < 1 || scratch == nullptr))) return FF_HOST_BAD_SHAPE;
  if (p.dk > 256) return FF_HOST_TOO_LARGE;
  const int heads = p.heads, dk = p.dk, dv = p.dv, tiles = p.tiles;
  const size_t items = (size_t)sequences * segments * heads;
  MlstmSegments sg = {segments, seg_len, 0, scratch, scratch + items * dk * dv, nullptr, nullptr, nullptr};
  sg.m_own = sg.n + items * tiles * dk;
  sg.f_own = sg.m_own + items * tiles;
  sg.m_start = sg.f_own + items * tiles;
  auto go = [&](auto kern, int bytes) -> int {
    const int smem = bytes + 128;
    if (int r = opt_in_smem(kern, smem)) return r;
    const dim3 grid(tiles, heads, sequences * segments);
    if (segments > 1) {
      sg.pass = 1;
      if (int r = launch_pdl(kern, grid, dim3(256), smem, s, 0, p, sg)) return r;
      const int sb = (dk * dv / 4 + 255) / 256, nb = SSD ? 0 : (tiles * dk / 4 + 255) / 256;
      if (int r = launch_pdl(mlstm_scan_kernel<SSD>, dim3(sb + nb, heads, sequences), dim3(256), 0, s, 0, p, sg, sb)) return r;
      sg.pass = 2;
    }
    if (int r = launch_pdl(kern, grid, dim3(256), smem, s, 0, p, sg)) return r;
    return launch_result();
  };
  if (dk <= 64) return go(mlstm_chunk_kernel<64, SSD>, (int)sizeof(MlstmSmem<64>));
  if (dk <= 128) return go(mlstm_chunk_kernel<128, SSD>, (int)sizeof(MlstmSmem<128>));
  return go(mlstm_chunk_kernel<256, SSD>, (int)sizeof(MlstmSmem<256>));
}

}  // namespace ff
using namespace ff;

// x: packed rows [rows, ldx]; gates FP32 [rows, ldg]; state and outputs as in MlstmArgs; row_start int[sequences + 1], slots
// int[sequences]. Rows are BF16 or FP32.
FF_EXPORT int ff_mlstm_recurrent(const void* x, const float* gates, const float* gate_bias, float* S, float* n, float* m, float* out,
                                 const int* row_start, const int* slots, int sequences, int ldx, int ldg, int heads, int dk, int dv, int tiles,
                                 float qscale, float cap, int f32, cudaStream_t s) {
  if (f32)
    return mlstm_recurrent_launch<false>(MlstmArgs<float>{(const float*)x, gates, gate_bias, S, n, m, out, row_start, slots, ldx, ldg, heads, dk, dv, tiles, qscale, cap, heads}, sequences, s);
  return mlstm_recurrent_launch<false>(MlstmArgs<__nv_bfloat16>{(const __nv_bfloat16*)x, gates, gate_bias, S, n, m, out, row_start, slots, ldx, ldg, heads, dk, dv, tiles, qscale, cap, heads}, sequences, s);
}

// Chunked form (BF16 rows, dk <= 256); segments, seg_len and scratch as in mlstm_chunked_launch
FF_EXPORT int ff_mlstm_chunked(const void* x, const float* gates, const float* gate_bias, float* S, float* n, float* m, float* out,
                               const int* row_start, const int* slots, int sequences, int ldx, int ldg, int heads, int dk, int dv, int tiles,
                               float qscale, float cap, int segments, int seg_len, float* scratch, cudaStream_t s) {
  const MlstmArgs<__nv_bfloat16> p = {(const __nv_bfloat16*)x, gates, gate_bias, S, n, m, out, row_start, slots, ldx, ldg, heads, dk, dv, tiles, qscale, cap, heads};
  return mlstm_chunked_launch<false>(p, sequences, segments, seg_len, scratch, s);
}

// State space. x: packed rows [C of the groups | B of the groups | x of the heads]; steps: logits [rows, lds] in the rows' type;
// bias, a, skip FP32 [heads]; S FP32 [slots, heads, dk, dv]; out FP32 [rows, heads, dv]
FF_EXPORT int ff_ssd_recurrent(const void* x, const void* steps, const float* bias, const float* a, const float* skip, float* S, float* out,
                               const int* row_start, const int* slots, int sequences, int ldx, int lds, int heads, int groups, int dk, int dv,
                               int f32, cudaStream_t s) {
  const int tiles = (dv + ML_TILE - 1) / ML_TILE;
  if (f32)
    return mlstm_recurrent_launch<true>(MlstmArgs<float>{(const float*)x, nullptr, bias, S, nullptr, nullptr, out, row_start, slots, ldx, lds, heads, dk, dv, tiles, 1.0f, 1.0f, groups, (const float*)steps, a, skip}, sequences, s);
  return mlstm_recurrent_launch<true>(MlstmArgs<__nv_bfloat16>{(const __nv_bfloat16*)x, nullptr, bias, S, nullptr, nullptr, out, row_start, slots, ldx, lds, heads, dk, dv, tiles, 1.0f, 1.0f, groups, (const __nv_bfloat16*)steps, a, skip}, sequences, s);
}

FF_EXPORT int ff_ssd_chunked(const void* x, const void* steps, const float* bias, const float* a, const float* skip, float* S, float* out,
                             const int* row_start, const int* slots, int sequences, int ldx, int lds, int heads, int groups, int dk, int dv,
                             int segments, int seg_len, float* scratch, cudaStream_t s) {
  const int tiles = (dv + ML_TILE - 1) / ML_TILE;
  const MlstmArgs<__nv_bfloat16> p = {(const __nv_bfloat16*)x, nullptr, bias, S, nullptr, nullptr, out, row_start, slots, ldx, lds, heads, dk, dv, tiles, 1.0f, 1.0f, groups, (const __nv_bfloat16*)steps, a, skip};
  return mlstm_chunked_launch<true>(p, sequences, segments, seg_len, scratch, s);
}

// o FP32 [rows, heads, dv] of which vdim elements of a head count; z rows of pitch ldz and w FP32 [heads * dv] laid out the same way;
// parts: equal pieces of the heads * vdim elements that are normed each by itself; y [rows, heads * dv]
FF_EXPORT int ff_ssd_out(const float* o, const void* z, int ldz, const float* w, void* y, int rows, int heads, int vdim, int dv, int parts, float eps,
                         int f32, cudaStream_t s) {
  if (rows <= 0 || rows > (1 << 30) || heads <= 0 || vdim <= 0 || dv < vdim || dv % 8 || parts < 1 || heads * vdim % parts || ldz < heads * dv) return FF_HOST_BAD_SHAPE;
  if (ldz % 8 || (reinterpret_cast<uintptr_t>(z) & 15) || (reinterpret_cast<uintptr_t>(w) & 15) || (reinterpret_cast<uintptr_t>(y) & 15)) return FF_HOST_BAD_ALIGN;
  if (rows > 65535) return FF_HOST_TOO_LARGE;
  const int part = heads * vdim / parts, smem = part * 4;
  if (smem > 200 * 1024) return FF_HOST_TOO_LARGE;
  int threads = (part / 4 + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 256 ? 256 : threads);
  auto go = [&](auto kern, auto zp, auto yp) -> int {
    if (int r = opt_in_smem(kern, smem)) return r;
    if (int r = launch_pdl(kern, dim3(parts, rows), dim3(threads), smem, s, 0, o, zp, ldz, w, yp, heads, vdim, dv, part, eps)) return r;
    return launch_result();
  };
  return f32 ? go(ssd_out_kernel<float>, (const float*)z, (float*)y) : go(ssd_out_kernel<__nv_bfloat16>, (const __nv_bfloat16*)z, (__nv_bfloat16*)y);
}

// o FP32 [rows, heads, dv]; gate [rows, heads * dv] with row pitch ldg; w FP32 [heads * dv]; y [rows, heads * dv]
FF_EXPORT int ff_mlstm_out(const float* o, const void* gate, int ldg, const float* w, void* y, int rows, int heads, int vdim, int dv, float eps,
                           int f32, cudaStream_t s) {
  if (rows <= 0 || heads <= 0 || vdim <= 0 || dv < vdim || dv % 16) return FF_HOST_BAD_SHAPE;
  if (ldg % 8 || (reinterpret_cast<uintptr_t>(gate) & 15) || (reinterpret_cast<uintptr_t>(w) & 15)) return FF_HOST_BAD_ALIGN;
  const dim3 grid((unsigned)(((long long)rows * heads + 7) / 8));
  const int r = f32 ? launch_pdl(mlstm_out_kernel<float>, grid, dim3(256), 0, s, 0, o, (const float*)gate, ldg, w, (float*)y, rows, heads, vdim, dv, eps)
                    : launch_pdl(mlstm_out_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, 0, o, (const __nv_bfloat16*)gate, ldg, w, (__nv_bfloat16*)y, rows, heads, vdim, dv, eps);
  return r ? r : launch_result();
}
