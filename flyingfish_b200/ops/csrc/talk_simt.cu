// Windowed attention whose heads' weights are mixed before they meet the values, on the CUDA cores: any head width, BF16 or FP32 (the
// tensor-core forms are in talk_tc.cu).
//   w_g(i, j) = exp(s_g(i, j)) / (one + sum_j exp(s_g(i, j)))        s_g(i, j) = scale (q_g(i) . k(j)),  0 <= i - j < window
//   o_h(i) = sum_j (sum_g talk[h, g] w_g(i, j)) v(j)                 v: the values of head h's own key / value head
// A block owns a query row with all its heads: a first pass over the visible keys finds every head's maximum and sum, a second one works
// out the weights of 32 keys at a time for all heads, mixes them and adds the values up. Everything in FP32.
#include "dtype_io.cuh"
#include "host_util.h"

namespace ff {

constexpr int TS_THREADS = 256, TS_KEYS = 32;

template <typename T>
struct TalkSimtArgs {
  const T* q; const T* kcache; const T* vcache;
  const int* block_table; const int* q_start; const int* q_lens; const int* ctx_lens;
  const float* talk; T* out;
  int batch, nq, hq, hkv, dk, dv, ldq, ldo, page, max_blocks, num_blocks, window;
  float scale, one;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(TS_THREADS)
talk_simt_kernel(const TalkSimtArgs<T> p) {
  pdl_trigger();
  extern __shared__ __align__(16) float ts[];
  float* sq = ts;                                          // [hq][dk]
  float* sp = sq + p.hq * p.dk;                            // [hq][32] weights, unmixed
  float* sm = sp + p.hq * TS_KEYS;                         // [hq][32] mixed
  float* st = sm + p.hq * TS_KEYS;                         // [hq][hq]
  float* acc = st + p.hq * p.hq;                           // [hq][dv]
  float* s_m = acc + p.hq * p.dv;                          // [hq] maximum, [hq] 1 / sum
  __shared__ int s_base[TS_KEYS], s_seq;
  const int row = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, H = p.hq, per = H / p.hkv;
  if (tid == 0) s_seq = -1;
  pdl_wait();
  __syncthreads();
  if (p.q_start == nullptr) { if (tid == 0) s_seq = row / p.nq; }
  else for (int i = tid; i < p.batch; i += TS_THREADS) if (row >= p.q_start[i] && row < p.q_start[i] + p.q_lens[i]) s_seq = i;
  __syncthreads();
  const int b = s_seq;
  const int at = b < 0 ? 0 : (p.q_start == nullptr ? row - b * p.nq : row - p.q_start[b]), len = b < 0 ? 0 : (p.q_start == nullptr ? p.nq : p.q_lens[b]);
  const int ctx = b < 0 ? 0 : p.ctx_lens[b], pos = ctx - len + at;
  for (int i = tid; i < H * p.dv; i += TS_THREADS) acc[i] = 0.f;
  if (ctx > 0 && pos >= 0) {                               // uniform in the block
    for (int i = tid; i < H * p.dk; i += TS_THREADS) sq[i] = to_float(p.q[(size_t)row * p.ldq + i]) * p.scale;
    for (int i = tid; i < H * H; i += TS_THREADS) st[i] = p.talk[i];
    const int lo = max(0, pos - p.window + 1);
    for (int pass = 0; pass < 2; ++pass) {
      float mx[8], sum[8];                                 // of heads warp, warp + 8, ...
#pragma unroll
      for (int i = 0; i < 8; ++i) { mx[i] = -INFINITY; sum[i] = 0.f; }
      for (int k0 = lo; k0 <= pos; k0 += TS_KEYS) {
        __syncthreads();                                   // the previous keys' places and weights have been read
        if (tid < TS_KEYS) {
          const int key = k0 + tid;
          int base = -1;
          if (key <= pos) {
            const int blk = p.block_table[(size_t)b * p.max_blocks + key / p.page];
            if (blk < 0 || blk >= p.num_blocks) set_status(p.status, KID_ATTN_DECODE, FF_ERR_BOUNDS, b, key);
            else base = blk * p.hkv * p.page + key % p.page;
          }
          s_base[tid] = base;
        }
        __syncthreads();
        const int base = s_base[lane];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int h = warp + 8 * i;
          if (h >= H) continue;
          float s = -INFINITY;
          if (base >= 0) {
            const T* kp = p.kcache + ((size_t)base + (size_t)(h / per) * p.page) * p.dk;
            float dot = 0.f;
            for (int d = 0; d < p.dk; d += 4) {
              float kv[4];
              load4(kp + d, kv);
              const float4 qv = *reinterpret_cast<const float4*>(sq + h * p.dk + d);
              dot = fmaf(qv.x, kv[0], dot); dot = fmaf(qv.y, kv[1], dot); dot = fmaf(qv.z, kv[2], dot); dot = fmaf(qv.w, kv[3], dot);
            }
            s = dot;
          }
          if (pass == 0) {
            const float mn = fmaxf(mx[i], warp_max(s));
            if (mn > -INFINITY) {
              sum[i] = sum[i] * expf(mx[i] - mn) + warp_sum(expf(s - mn));
              mx[i] = mn;
            }
          } else {
            sp[h * TS_KEYS + lane] = expf(s - s_m[h]) * s_m[H + h];
          }
        }
        if (pass == 0) continue;
        __syncthreads();
        for (int i = tid; i < H * TS_KEYS; i += TS_THREADS) {
          const int h = i / TS_KEYS, j = i - h * TS_KEYS;
          float w = 0.f;
          for (int g = 0; g < H; ++g) w = fmaf(st[h * H + g], sp[g * TS_KEYS + j], w);
          sm[i] = w;
        }
        __syncthreads();
        for (int i = tid; i < H * p.dv; i += TS_THREADS) { // a thread's own sums in every round
          const int h = i / p.dv, c = i - h * p.dv;
          float a = acc[i];
          for (int j = 0; j < TS_KEYS; ++j)
            if (s_base[j] >= 0) a = fmaf(sm[h * TS_KEYS + j], to_float(p.vcache[((size_t)s_base[j] + (size_t)(h / per) * p.page) * p.dv + c]), a);
          acc[i] = a;
        }
      }
      if (pass == 0) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int h = warp + 8 * i;
          if (h >= H || lane != 0) continue;
          const float m = p.one > 0.f ? fmaxf(mx[i], 0.f) : mx[i];
          s_m[h] = m;
          s_m[H + h] = m > -INFINITY ? 1.0f / (sum[i] * expf(mx[i] - m) + p.one * expf(-m)) : 0.f;
        }
        __syncthreads();
      }
    }
  }
  __syncthreads();
  for (int i = tid; i < H * p.dv; i += TS_THREADS) from_float(p.out + (size_t)row * p.ldo + i, acc[i]);
}

template <typename T>
static int talk_simt_launch(const TalkSimtArgs<T>& p, int rows, cudaStream_t s) {
  const int smem = (p.hq * (p.dk + 2 * TS_KEYS + p.hq + p.dv) + 2 * p.hq) * 4;
  if (smem > 200 * 1024) return FF_HOST_TOO_LARGE;
  if (int r = opt_in_smem(talk_simt_kernel<T>, smem)) return r;
  if (int r = launch_pdl(talk_simt_kernel<T>, dim3(rows), dim3(TS_THREADS), smem, s, 0, p)) return r;
  return launch_result();
}

}  // namespace ff
using namespace ff;

// q rows of pitch ldq (heads dk wide); caches [blocks, hkv, page, dk / dv]; talk FP32 [hq, hq]; out rows of pitch ldo (heads dv wide). Rows
// come as ranges (q_start / q_lens) or nq per sequence; one: the soft-max's extra term in the denominator (0 or 1).
FF_EXPORT int ff_talk_simt(const void* q, const void* kcache, const void* vcache, const int* block_table, const int* q_start, const int* q_lens,
                           const int* ctx_lens, const float* talk, void* out, int batch, int rows, int nq, int hq, int hkv, int dk, int dv, int ldq,
                           int ldo, int page, int max_blocks, int num_blocks, int window, float scale, float one, int f32, int* status,
                           cudaStream_t s) {
  if (batch <= 0 || rows <= 0 || nq < 1 || hq <= 0 || hq > 64 || hkv <= 0 || hq % hkv || dk <= 0 || dk % 4 || dv <= 0 || page <= 0 || window < 1) return FF_HOST_BAD_SHAPE;
  if ((q_start == nullptr) != (q_lens == nullptr) || (q_start == nullptr && rows != batch * nq) || !(one >= 0.f)) return FF_HOST_BAD_SHAPE;
  if (f32)
    return talk_simt_launch(TalkSimtArgs<float>{(const float*)q, (const float*)kcache, (const float*)vcache, block_table, q_start, q_lens, ctx_lens, talk, (float*)out, batch, nq, hq, hkv, dk, dv, ldq, ldo, page, max_blocks, num_blocks, window, scale, one, status}, rows, s);
  return talk_simt_launch(TalkSimtArgs<__nv_bfloat16>{(const __nv_bfloat16*)q, (const __nv_bfloat16*)kcache, (const __nv_bfloat16*)vcache, block_table, q_start, q_lens, ctx_lens, talk, (__nv_bfloat16*)out, batch, nq, hq, hkv, dk, dv, ldq, ldo, page, max_blocks, num_blocks, window, scale, one, status}, rows, s);
}
