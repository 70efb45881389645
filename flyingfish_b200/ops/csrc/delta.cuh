// What the kernels of the channel-wise gated delta rule share: their arguments and the FP32 gates.
#pragma once
#include "dtype_io.cuh"

namespace ff {

constexpr int DL_TILE = 64;           // value columns a CTA owns

template <typename T>
struct DeltaArgs {
  const T* x;                         // packed convolved rows: q at g * dk, k at (G + g) * dk, v at 2 G dk + h * dv
  const float* unit;                  // [rows, 2 G]: factors that make q and k unit vectors (q's with its scale)
  const float* decay;                 // [rows, ldd]: logits of the decays, head h at h * dk
  const T* beta;                      // [rows, ldb]: logits of the step sizes
  const float* rate;                  // [H]: -exp(A_log)
  const float* dt_bias;               // [H * dk]
  float* S;                           // [slots, H, dk, dv]
  float* out;                         // [rows, H, dv]
  const int* row_start; const int* slots;
  int ldx, ldd, ldb, heads, kv_heads, dk, dv;
};

// logarithm of a decay
__device__ __forceinline__ float log_decay(float logit, float bias, float rate) {
  const float z = logit + bias;
  return rate * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))));
}

}  // namespace ff
