// Warp-level mma.sync m16n8k16 (BF16 x BF16 -> FP32) and ldmatrix helpers for small attention tiles whose operands are
// produced in shared memory by the CTA itself (de-quantised cache rows), where a tcgen05 pipeline has nothing to stream.
#pragma once
#include <cstdint>
#include "ptx.cuh"

namespace ff {

__device__ __forceinline__ void ms_ldsm4(uint32_t a, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void ms_ldsm4t(uint32_t a, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void ms_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// byte offset of 16-byte chunk c of row r in a [rows][chunks * 8] bf16 tile whose chunk index is XORed with r % 8
__device__ __forceinline__ uint32_t ms_off(int r, int c, int chunks) { return (uint32_t)((r * chunks + ((c & ~7) | ((c ^ r) & 7))) * 16); }


// store a pair of accumulator values as BF16 at (row, col .. col+1) of a swizzled tile with `chunks` 16-byte chunks per row
__device__ __forceinline__ void ms_store2(uint8_t* tile, int row, int col, int chunks, float x, float y) {
  *reinterpret_cast<uint32_t*>(tile + ms_off(row, col >> 3, chunks) + (col & 7) * 2) = pack_bf16x2(x, y);
}

// acc[NT][4] (+)= A[m0 .. m0+15][0 .. 16 KS) . B, A row-major tile (a_chunks per row);
// B_TRANS = false: B given as [n][k] rows (b_chunks per row), n-tiles n0 .. n0 + 8 NT
// B_TRANS = true : B given as [k][n] rows, same n range
template <int NT, int KS, bool B_TRANS>
__device__ __forceinline__ void ms_product(float (&acc)[NT][4], uint32_t a_base, int a_chunks, int m0, uint32_t b_base, int b_chunks,
                                        int n0, int lane) {
#pragma unroll
  for (int ks = 0; ks < KS; ++ks) {
    uint32_t a[4];
    ms_ldsm4(a_base + ms_off(m0 + (lane & 7) + (((lane >> 3) & 1) << 3), 2 * ks + (lane >> 4), a_chunks), a[0], a[1], a[2], a[3]);
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) {
      uint32_t b0, b1, b2, b3;
      if (B_TRANS) {
        const int krow = ks * 16 + (((lane >> 3) & 1) << 3) + (lane & 7);
        ms_ldsm4t(b_base + ms_off(krow, (n0 >> 3) + 2 * np + (lane >> 4), b_chunks), b0, b1, b2, b3);
      } else {
        ms_ldsm4(b_base + ms_off(n0 + 16 * np + ((lane >> 4) << 3) + (lane & 7), 2 * ks + ((lane >> 3) & 1), b_chunks), b0, b1, b2, b3);
      }
      ms_mma(acc[2 * np], a, b0, b1);
      ms_mma(acc[2 * np + 1], a, b2, b3);
    }
  }
}

}  // namespace ff
