// Paged attention on the CUDA cores, for what the tensor-core kernels do not take: FP32 caches and head widths above 128.
// One warp per (query row, head): 32 keys at a time, a key per lane for the scores, a channel per lane for the values,
// soft-max and accumulation in FP32 (online). Causal, sliding window (that may keep the first positions), block-local (`chunk`) or
// bidirectional; optional capped scores, output gate (per element or per head) and sinks. Rows come as ranges (q_start / q_lens; chunked prefill) or nq per sequence (decode).
#include "dtype_io.cuh"
#include "host_util.h"
#include <climits>

namespace ff {

constexpr int AS_WARPS = 4;

template <typename T, int NV>          // NV: value channels per lane
__global__ void __launch_bounds__(32 * AS_WARPS)
attn_simt_kernel(const T* __restrict__ q, const T* __restrict__ kcache, const T* __restrict__ vcache, const int* __restrict__ block_table,
                 const int* __restrict__ q_start, const int* __restrict__ q_lens, const int* __restrict__ ctx_lens, T* __restrict__ out,
                 int batch, int rows, int nq, int hq, int hkv, int dk, int dv, int ldq, int ldo, int page, int max_blocks,
                 int num_blocks, float scale, int window, int chunk, const T* __restrict__ gate, int ldg, const float* __restrict__ sinks, int* status,
                 int ldv, int keep, float softcap, int head_gate) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) float as_q[];            // [AS_WARPS][dk]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * AS_WARPS + warp;
  if (item >= (long long)rows * hq) return;
  const int row = (int)(item / hq), h = (int)(item % hq), g = h / (hq / hkv);
  // sequence of the row and the row's place in it
  int b = -1, at = 0, qlen = nq;
  if (q_start == nullptr) {
    b = row / nq; at = row - b * nq;
  } else {
    for (int i = lane; i < batch; i += 32)
      if (row >= q_start[i] && row < q_start[i] + q_lens[i]) b = i;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) b = max(b, __shfl_xor_sync(0xffffffffu, b, o));
    if (b >= 0) { at = row - q_start[b]; qlen = q_lens[b]; }
  }
  const int ctx = b >= 0 && b < batch ? ctx_lens[b] : 0;
  const int pos = ctx - qlen + at;
  float acc[NV];
#pragma unroll
  for (int j = 0; j < NV; ++j) acc[j] = 0.f;
  float m = -INFINITY, l = 0.f;
  if (ctx > 0 && pos >= 0) {
    float* sq = as_q + warp * dk;
    for (int d = lane; d < dk; d += 32) sq[d] = to_float(q[(size_t)row * ldq + (size_t)h * dk + d]);
    __syncwarp();
    const int hi = window < 0 ? ctx - 1 : pos;
    const int lo = window > 0 ? max(0, pos - window + 1) : (chunk > 0 ? pos / chunk * chunk : 0);
    const int kept = min(keep, lo), front = (kept + 31) / 32 * 32;      // kept positions before the window come first
    for (int k0 = -front; k0 <= hi - lo; k0 += 32) {
      const int at = k0 + front + lane;
      const int key = k0 >= 0 ? lo + k0 + lane : (at < kept ? at : INT_MAX);
      float s = -INFINITY;
      int base = -1;                                       // (block * hkv + kv head) * page + offset
      if (key <= hi) {
        const int blk = block_table[(size_t)b * max_blocks + key / page];
        if (blk < 0 || blk >= num_blocks) set_status(status, KID_ATTN_DECODE, FF_ERR_BOUNDS, b, key);
        else {
          base = (blk * hkv + g) * page + key % page;
          const T* kp = kcache + (size_t)base * dk;
          float dot = 0.f;
          for (int d = 0; d < dk; d += 4) {
            float kv[4];
            load4(kp + d, kv);
            const float4 qv = *reinterpret_cast<const float4*>(sq + d);
            dot = fmaf(qv.x, kv[0], dot); dot = fmaf(qv.y, kv[1], dot); dot = fmaf(qv.z, kv[2], dot); dot = fmaf(qv.w, kv[3], dot);
          }
          s = dot * scale;
          if (softcap > 0.f) s = softcap * tanhf(s / softcap);
        }
      }
      const float mn = fmaxf(m, warp_max(s));
      if (mn == -INFINITY) continue;
      const float alpha = expf(m - mn), p = expf(s - mn);
      m = mn;
      l = l * alpha + warp_sum(p);
#pragma unroll
      for (int j = 0; j < NV; ++j) acc[j] *= alpha;
      for (int i = 0; i < 32; ++i) {
        const float pi = __shfl_sync(0xffffffffu, p, i);
        const int bi = __shfl_sync(0xffffffffu, base, i);
        if (bi < 0) continue;
        const T* vp = vcache + (size_t)bi * ldv;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          const int c = lane + 32 * j;
          if (c < dv) acc[j] = fmaf(pi, to_float(vp[c]), acc[j]);
        }
      }
    }
  }
  // learnable soft-max: the head's sink logit enters the denominator only
  if (sinks != nullptr && m > -INFINITY) {
    const float sk = sinks[h], mn = fmaxf(m, sk), a = expf(m - mn);
    l = l * a + expf(sk - mn);
#pragma unroll
    for (int j = 0; j < NV; ++j) acc[j] *= a;
  }
  const float inv = l > 0.f ? 1.0f / l : 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int c = lane + 32 * j;
    if (c < dv) {
      float o = acc[j] * inv;
      if (gate != nullptr) o *= sigmoid_f(to_float(gate[(size_t)row * ldg + (head_gate ? (size_t)h : (size_t)h * dv + c)]));
      from_float(out + (size_t)row * ldo + (size_t)h * dv + c, o);
    }
  }
}

template <typename T>
static int attn_simt_launch(const void* q, const void* kc, const void* vc, const int* bt, const int* q_start, const int* q_lens,
                            const int* ctx_lens, void* out, int batch, int rows, int nq, int hq, int hkv, int dk, int dv, int ldq, int ldo,
                            int page, int max_blocks, int num_blocks, float scale, int window, int chunk, const void* gate, int ldg,
                            const float* sinks, int* status, int ldv, int keep, float softcap, int head_gate, cudaStream_t s) {
  const long long blocks = ((long long)rows * hq + AS_WARPS - 1) / AS_WARPS;
  const int smem = AS_WARPS * dk * 4;
  auto go = [&](auto kern) -> int {
    if (int r = opt_in_smem(kern, smem)) return r;
    if (int r = launch_pdl(kern, dim3((unsigned)blocks), dim3(32 * AS_WARPS), smem, s, 0, (const T*)q, (const T*)kc, (const T*)vc, bt, q_start, q_lens,
                           ctx_lens, (T*)out, batch, rows, nq, hq, hkv, dk, dv, ldq, ldo, page, max_blocks, num_blocks, scale, window, chunk,
                           (const T*)gate, ldg, sinks, status, ldv, keep, softcap, head_gate)) return r;
    return launch_result();
  };
  if (dv <= 128) return go(attn_simt_kernel<T, 4>);
  if (dv <= 512) return go(attn_simt_kernel<T, 16>);
  if (dv <= 1024) return go(attn_simt_kernel<T, 32>);
  return FF_HOST_TOO_LARGE;
}

}  // namespace ff
using namespace ff;

// window > 0 sliding (the first `keep` positions stay visible), < 0 bidirectional, 0 causal; chunk > 0: keys of the query's own block of
// `chunk` positions; ldv: pitch of the value cache's rows; softcap > 0: scores become softcap tanh(score / softcap); head_gate: the
// gate has one column per head
FF_EXPORT int ff_attn_simt(const void* q, const void* kcache, const void* vcache, const int* block_table, const int* q_start,
                           const int* q_lens, const int* ctx_lens, void* out, int batch, int rows, int nq, int hq, int hkv, int dk, int dv,
                           int ldq, int ldo, int page, int max_blocks, int num_blocks, float scale, int window, int chunk, const void* gate,
                           int ldg, const float* sinks, int f32, int* status, int ldv, int keep, float softcap, int head_gate, cudaStream_t s) {
  if (ldv < dv || keep < 0 || !(softcap >= 0.f)) return FF_HOST_BAD_SHAPE;
  if (window <= 0) keep = 0;
  if (batch <= 0 || rows <= 0 || nq < 1 || hq <= 0 || hkv <= 0 || hq % hkv || dk <= 0 || dk % 4 || dv <= 0 || page <= 0 || chunk < 0)
    return FF_HOST_BAD_SHAPE;
  if ((q_start == nullptr) != (q_lens == nullptr) || (q_start == nullptr && rows != batch * nq)) return FF_HOST_BAD_SHAPE;
  if (window != 0 && chunk > 0) return FF_HOST_UNSUPPORTED;
  if (f32) return attn_simt_launch<float>(q, kcache, vcache, block_table, q_start, q_lens, ctx_lens, out, batch, rows, nq, hq, hkv, dk, dv, ldq, ldo, page, max_blocks, num_blocks, scale, window, chunk, gate, ldg, sinks, status, ldv, keep, softcap, head_gate, s);
  return attn_simt_launch<__nv_bfloat16>(q, kcache, vcache, block_table, q_start, q_lens, ctx_lens, out, batch, rows, nq, hq, hkv, dk, dv, ldq, ldo, page, max_blocks, num_blocks, scale, window, chunk, gate, ldg, sinks, status, ldv, keep, softcap, head_gate, s);
}
