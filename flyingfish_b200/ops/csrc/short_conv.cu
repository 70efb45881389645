// Short causal convolution per channel in front of a recurrence, with its last inputs carried per sequence:
//   y[t, c] = silu(b[c] + sum_j w[j, c] x[t - (TAPS - 1) + j, c])
// Rows before a sequence's first new one come from its history (zero at the start), which then takes the last TAPS - 1 inputs. The
// channels are heads: `nh` of them `dn` wide and then `vh` of them `dv` wide. For the first `nh` the kernel also writes
// factor / sqrt(sum of squares + 1e-6) of the result as stored (unit vectors), `factor` being `qscale` for the first half of them.
// A group of G lanes owns a head and up to CV_ROWS consecutive rows; the inputs it needs stay in registers.
#include "dtype_io.cuh"
#include "host_util.h"
#include <type_traits>

namespace ff {

constexpr int CV_THREADS = 128;
constexpr int CV_ROWS = 16;           // rows of a tile; at least the largest TAPS - 1, so that only a sequence's first tile reads history

template <typename T>
struct ConvArgs {
  const T* x; T* y; const float* w; const float* bias;     // w [TAPS][channels]
  float* history;                                          // [slots][TAPS - 1][channels]
  float* unit;                                             // [rows, nh] or null
  const int* row_start; const int* slots;
  int ldx, channels, nh, dn, vh, dv, tiles;
  float qscale;
};

__device__ __forceinline__ float conv_silu(float v, __nv_bfloat16) { return __fdividef(v, 1.0f + __expf(-v)); }
__device__ __forceinline__ float conv_silu(float v, float) { return v * sigmoid_f(v); }
__device__ __forceinline__ float stored(float v, __nv_bfloat16) { return __bfloat162float(__float2bfloat16(v)); }
__device__ __forceinline__ float stored(float v, float) { return v; }

// NV: vectors of 8 channels a lane holds
template <typename T, int TAPS, int G, int NV>
__global__ void __launch_bounds__(CV_THREADS)
short_conv_kernel(const ConvArgs<T> p) {
  pdl_trigger();
  pdl_wait();
  const int seq = blockIdx.y, gl = threadIdx.x & (G - 1);
  const int item = blockIdx.x * (CV_THREADS / G) + threadIdx.x / G;
  const int heads = p.nh + p.vh, head = item % heads, tile = item / heads;
  const int r0 = p.row_start[seq], n = p.row_start[seq + 1] - r0, t0 = tile * CV_ROWS;
  const bool live = tile < p.tiles && t0 < n;              // uniform in a group; its lanes stay for the shuffles
  const bool normed = head < p.nh;
  const int d = normed ? p.dn : p.dv, base = normed ? head * p.dn : p.nh * p.dn + (head - p.nh) * p.dv;
  float* hist = p.history + (size_t)p.slots[seq] * (TAPS - 1) * p.channels;
  float win[NV][TAPS][8], w[NV][TAPS][8], b[NV][8];
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int c = (gl + v * G) * 8, ch = base + c;
    const bool on = live && c < d;
#pragma unroll
    for (int i = 0; i < 8; ++i) b[v][i] = 0.f;
    if (on && p.bias != nullptr) load8(p.bias + ch, b[v]);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
#pragma unroll
      for (int i = 0; i < 8; ++i) { win[v][j][i] = 0.f; w[v][j][i] = 0.f; }
      if (!on) continue;
      load8(p.w + (size_t)j * p.channels + ch, w[v][j]);
      const int t = t0 - (TAPS - 1) + j;                   // the inputs before the tile's first row: 0 .. TAPS - 2
      if (j < TAPS - 1) {
        if (t >= 0) load8(p.x + (size_t)(r0 + t) * p.ldx + ch, win[v][j]);
        else load8(hist + (size_t)(t + TAPS - 1) * p.channels + ch, win[v][j]);
      }
    }
  }
  const int rows = live ? min(CV_ROWS, n - t0) : 0;
  if (live && tile == 0 && TAPS > 1) {
    // the next call's history, before anything of this one is overwritten: a thread reads and writes its own channels only
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int c = (gl + v * G) * 8, ch = base + c;
      if (c >= d) continue;
      float next[TAPS > 1 ? TAPS - 1 : 1][8];
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int t = n - (TAPS - 1) + j;
        if (t >= 0) load8(p.x + (size_t)(r0 + t) * p.ldx + ch, next[j]);
        else load8(hist + (size_t)(t + TAPS - 1) * p.channels + ch, next[j]);
      }
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) store8(hist + (size_t)j * p.channels + ch, next[j]);
    }
  }
  for (int r = 0; r < CV_ROWS; ++r) {
    if (!__any_sync(0xffffffffu, r < rows)) break;
    float ss = 0.f;
    const size_t row = (size_t)(r0 + t0 + r);
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int c = (gl + v * G) * 8, ch = base + c;
      if (r >= rows || c >= d) continue;
      load8(p.x + row * p.ldx + ch, win[v][TAPS - 1]);
      float y[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        float a = b[v][i];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) a = fmaf(w[v][j][i], win[v][j][i], a);
        y[i] = stored(conv_silu(a, T()), T());
        ss = fmaf(y[i], y[i], ss);
      }
      store8(p.y + row * p.channels + ch, y);
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
        for (int i = 0; i < 8; ++i) win[v][j][i] = win[v][j + 1][i];
    }
    if (p.unit != nullptr) {
#pragma unroll
      for (int o = G / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o, G);
      if (gl == 0 && normed && r < rows) p.unit[row * p.nh + head] = (head < p.nh / 2 ? p.qscale : 1.0f) / sqrtf(ss + 1e-6f);
    }
  }
}

template <typename T>
static int short_conv_launch(const ConvArgs<T>& p, int taps, int sequences, cudaStream_t s) {
  const int vecs = (p.dn > p.dv ? p.dn : p.dv) / 8;
  auto go = [&](auto kern, int g) -> int {
    const long long blocks = ((long long)p.tiles * (p.nh + p.vh) * g + CV_THREADS - 1) / CV_THREADS;
    if (int r = launch_pdl(kern, dim3((unsigned)blocks, sequences), dim3(CV_THREADS), 0, s, 0, p)) return r;
    return launch_result();
  };
  auto width = [&](auto tag) -> int {
    constexpr int K = decltype(tag)::value;
    if (vecs <= 8) return go(short_conv_kernel<T, K, 8, 1>, 8);
    if (vecs <= 16) return go(short_conv_kernel<T, K, 16, 1>, 16);
    if (vecs <= 32) return go(short_conv_kernel<T, K, 32, 1>, 32);
    if (vecs <= 64) return go(short_conv_kernel<T, K, 32, 2>, 32);
    return FF_HOST_TOO_LARGE;
  };
  switch (taps) {
    case 1: return width(std::integral_constant<int, 1>{});
    case 2: return width(std::integral_constant<int, 2>{});
    case 3: return width(std::integral_constant<int, 3>{});
    case 4: return width(std::integral_constant<int, 4>{});
    case 5: return width(std::integral_constant<int, 5>{});
    case 6: return width(std::integral_constant<int, 6>{});
    case 7: return width(std::integral_constant<int, 7>{});
    case 8: return width(std::integral_constant<int, 8>{});
  }
  return FF_HOST_UNSUPPORTED;
}

}  // namespace ff
using namespace ff;

// x: rows of pitch ldx, y: rows of `channels` = nh * dn + vh * dv; w FP32 [taps, channels], bias FP32 [channels] or null; history FP32
// [slots, taps - 1, channels]; unit FP32 [rows, nh] or null; row_start int[sequences + 1], slots int[sequences]; max_rows: the longest
// sequence's rows.
FF_EXPORT int ff_short_conv(const void* x, void* y, const float* w, const float* bias, float* history, float* unit, const int* row_start,
                            const int* slots, int sequences, int max_rows, int ldx, int nh, int dn, int vh, int dv, int taps, float qscale, int f32,
                            cudaStream_t s) {
  const long long channels = (long long)nh * dn + (long long)vh * dv;
  if (sequences <= 0 || sequences > 65535 || max_rows <= 0 || nh < 0 || vh < 0 || nh + vh == 0 || dn < 0 || dv < 0 || dn % 8 || dv % 8) return FF_HOST_BAD_SHAPE;
  if ((nh > 0 && dn == 0) || (vh > 0 && dv == 0) || channels > (1 << 24) || ldx < channels) return FF_HOST_BAD_SHAPE;
  if (ldx % 8 || (reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(y) & 15) || (reinterpret_cast<uintptr_t>(history) & 15) ||
      (reinterpret_cast<uintptr_t>(w) & 15) || (reinterpret_cast<uintptr_t>(bias) & 15)) return FF_HOST_BAD_ALIGN;
  const int tiles = (max_rows + CV_ROWS - 1) / CV_ROWS;
  auto args = [&](auto* t) {
    using T = std::remove_pointer_t<decltype(t)>;
    return ConvArgs<T>{(const T*)x, (T*)y, w, bias, history, unit, row_start, slots, ldx, (int)channels, nh, dn, vh, dv, tiles, qscale};
  };
  if (f32) return short_conv_launch(args((float*)nullptr), taps, sequences, s);
  return short_conv_launch(args((__nv_bfloat16*)nullptr), taps, sequences, s);
}
