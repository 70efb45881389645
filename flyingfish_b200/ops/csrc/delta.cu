// Gated delta rule with a decay per key channel. Per head, with decays g_t in (0, 1]^dk on the rows of S [dk, dv]:
//   S <- diag(g_t) S        u_t = beta_t (v_t - S^T k_t)        S <- S + k_t u_t^T        o_t = S^T q_t
//   g_t = exp(-exp(A_log) softplus(z_t + dt_bias)),  beta_t = sigmoid(b_t),  q and k unit vectors
// recurrent : token by token in FP32, BF16 or FP32 rows (decode; 32-bit prompts). The state of 64 value columns sits in registers
//             while the tokens of a sequence pass; both products with the decayed state are one pass (o = S^T q + (q . k) u).
// out       : every head divided by its root mean square, times a weight and the sigmoid of a gate (delta_head_out).
// The form of prompts is in delta_chunk.cu.
#include "delta.cuh"
#include "host_util.h"

namespace ff {

// grid (tiles, heads, sequences), 256 threads = 16 float4 columns x 16 key groups; R key rows per thread
template <typename T, int R>
__global__ void __launch_bounds__(256)
delta_recurrent_kernel(const DeltaArgs<T> p) {
  pdl_trigger();
  pdl_wait();
  constexpr int KP = 16 * R;
  __shared__ float sq[2][KP], sk[2][KP], sg[2][KP];
  __shared__ __align__(16) float s_k[2][8][DL_TILE], s_q[2][8][DL_TILE];
  __shared__ float s_qk[2][8];
  const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r0 = p.row_start[seq], r1 = p.row_start[seq + 1];
  if (r1 <= r0) return;
  const int H = p.heads, G = p.kv_heads, g = h / (H / G), dk = p.dk, dv = p.dv;
  const int c = tid & 15, kg = tid >> 4, col = blockIdx.x * DL_TILE + c * 4;
  const bool live = col < dv;
  float* Sg = p.S + ((size_t)p.slots[seq] * H + h) * dk * dv + col;
  float st[R][4];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int k = kg + 16 * r;
    if (live && k < dk) load4(Sg + (size_t)k * dv, st[r]);
    else st[r][0] = st[r][1] = st[r][2] = st[r][3] = 0.f;
  }
  const float rate = p.rate[h];
  for (int row = r0; row < r1; ++row) {
    const int par = (row - r0) & 1;
    const T* xr = p.x + (size_t)row * p.ldx;
    const float fq = p.unit[(size_t)row * 2 * G + g], fk = p.unit[(size_t)row * 2 * G + G + g];
    const float beta = sigmoid_f(to_float(p.beta[(size_t)row * p.ldb + h]));
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (live) load4(xr + (size_t)2 * G * dk + (size_t)h * dv + col, v);
    float qk = 0.f;
    for (int k = tid; k < KP; k += 256) {
      float a = 0.f, b = 0.f, d = 0.f;
      if (k < dk) {
        a = to_float(xr[(size_t)g * dk + k]) * fq;
        b = to_float(xr[(size_t)(G + g) * dk + k]) * fk;
        d = expf(log_decay(p.decay[(size_t)row * p.ldd + (size_t)h * dk + k], p.dt_bias[(size_t)h * dk + k], rate));
      }
      sq[par][k] = a; sk[par][k] = b; sg[par][k] = d;
      qk = fmaf(a, b, qk);
    }
    qk = warp_sum(qk);
    if (lane == 0) s_qk[par][warp] = qk;
    __syncthreads();
    float ak[4] = {0.f, 0.f, 0.f, 0.f}, aq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int k = kg + 16 * r;
      const float d = sg[par][k], kk = sk[par][k], qq = sq[par][k];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        st[r][j] *= d;
        ak[j] = fmaf(kk, st[r][j], ak[j]);
        aq[j] = fmaf(qq, st[r][j], aq[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      ak[j] += __shfl_xor_sync(0xffffffffu, ak[j], 16);
      aq[j] += __shfl_xor_sync(0xffffffffu, aq[j], 16);
    }
    if (lane < 16) { store4(&s_k[par][warp][c * 4], ak); store4(&s_q[par][warp][c * 4], aq); }
    __syncthreads();
    float u[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      float t[4];
      load4(&s_k[par][w][c * 4], t);
#pragma unroll
      for (int j = 0; j < 4; ++j) u[j] += t[j];
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) u[j] = beta * (v[j] - u[j]);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const float kk = sk[par][kg + 16 * r];
#pragma unroll
      for (int j = 0; j < 4; ++j) st[r][j] = fmaf(kk, u[j], st[r][j]);
    }
    if (kg == 0 && live) {
      float o[4] = {0.f, 0.f, 0.f, 0.f}, dot = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        float t[4];
        load4(&s_q[par][w][c * 4], t);
        dot += s_qk[par][w];
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] += t[j];
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = fmaf(dot, u[j], o[j]);
      store4(p.out + ((size_t)row * H + h) * dv + col, o);
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int k = kg + 16 * r;
    if (live && k < dk) store4(Sg + (size_t)k * dv, st[r]);
  }
}

// out: one warp per (row, head): y = o / rms(o) * w * sigmoid(gate); the weight is shared by the heads
template <typename T>
__global__ void __launch_bounds__(256)
delta_out_kernel(const float* __restrict__ o, const T* __restrict__ gate, int ldg, const float* __restrict__ w, T* __restrict__ y, int rows,
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
    load4(w + c, f);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = v[j] * r * f[j] * sigmoid_f(g[j]);
    store4(y + item * dv + c, v);
  }
}

template <typename T>
static int delta_recurrent_launch(const DeltaArgs<T>& p, int sequences, cudaStream_t s) {
  auto go = [&](auto kern) -> int {
    if (int r = launch_pdl(kern, dim3((p.dv + DL_TILE - 1) / DL_TILE, p.heads, sequences), dim3(256), 0, s, 0, p)) return r;
    return launch_result();
  };
  if (p.dk <= 16) return go(delta_recurrent_kernel<T, 1>);
  if (p.dk <= 32) return go(delta_recurrent_kernel<T, 2>);
  if (p.dk <= 64) return go(delta_recurrent_kernel<T, 4>);
  if (p.dk <= 128) return go(delta_recurrent_kernel<T, 8>);
  if (p.dk <= 256) return go(delta_recurrent_kernel<T, 16>);
  if (p.dk <= 512) return go(delta_recurrent_kernel<T, 32>);
  return FF_HOST_TOO_LARGE;
}

}  // namespace ff
using namespace ff;

// Arguments as in DeltaArgs; row_start int[sequences + 1], slots int[sequences]. Rows are BF16 or FP32.
FF_EXPORT int ff_delta_recurrent(const void* x, const float* unit, const float* decay, const void* beta, const float* rate, const float* dt_bias,
                                 float* S, float* out, const int* row_start, const int* slots, int sequences, int ldx, int ldd, int ldb,
                                 int heads, int kv_heads, int dk, int dv, int f32, cudaStream_t s) {
  if (sequences <= 0 || sequences > 65535 || heads <= 0 || heads > 65535 || kv_heads <= 0 || heads % kv_heads || dk <= 0 || dk % 8 || dv <= 0 || dv % 8)
    return FF_HOST_BAD_SHAPE;
  if (ldx < 2 * kv_heads * dk + heads * dv || ldd < heads * dk || ldb < heads) return FF_HOST_BAD_SHAPE;
  if (ldx % 8 || (reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(S) & 15) || (reinterpret_cast<uintptr_t>(out) & 15)) return FF_HOST_BAD_ALIGN;
  if (f32)
    return delta_recurrent_launch(DeltaArgs<float>{(const float*)x, unit, decay, (const float*)beta, rate, dt_bias, S, out, row_start, slots, ldx, ldd, ldb, heads, kv_heads, dk, dv}, sequences, s);
  return delta_recurrent_launch(DeltaArgs<__nv_bfloat16>{(const __nv_bfloat16*)x, unit, decay, (const __nv_bfloat16*)beta, rate, dt_bias, S, out, row_start, slots, ldx, ldd, ldb, heads, kv_heads, dk, dv}, sequences, s);
}

// o FP32 [rows, heads, dv] of which vdim count; gate rows of pitch ldg; w FP32 [dv]; y [rows, heads * dv]
FF_EXPORT int ff_delta_out(const float* o, const void* gate, int ldg, const float* w, void* y, int rows, int heads, int vdim, int dv, float eps,
                           int f32, cudaStream_t s) {
  if (rows <= 0 || heads <= 0 || vdim <= 0 || dv < vdim || dv % 8) return FF_HOST_BAD_SHAPE;
  if (ldg % 8 || (reinterpret_cast<uintptr_t>(gate) & 15) || (reinterpret_cast<uintptr_t>(w) & 15)) return FF_HOST_BAD_ALIGN;
  const dim3 grid((unsigned)(((long long)rows * heads + 7) / 8));
  const int r = f32 ? launch_pdl(delta_out_kernel<float>, grid, dim3(256), 0, s, 0, o, (const float*)gate, ldg, w, (float*)y, rows, heads, vdim, dv, eps)
                    : launch_pdl(delta_out_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, 0, o, (const __nv_bfloat16*)gate, ldg, w, (__nv_bfloat16*)y, rows, heads, vdim, dv, eps);
  return r ? r : launch_result();
}
