// 16x16 tiles of mma.sync.m16n8k16 for the kernels that evaluate a linear recurrence a chunk of tokens at
// a time: operands out of shared memory, results to and from it, and the split of a float32 value into a
// bfloat16 head and remainder.
#pragma once

#include "attention_tiles.cuh"

// Operands of mma.sync.m16n8k16 out of shared memory by ldmatrix, for a 16x16 tile of the result (two
// blocks of 8 columns: b[0], b[1] feed the first, b[2], b[3] the second).  "rows": the tile lies
// as it is multiplied (A as [m][k], B as [k][n]); "cols": it lies transposed (A as [k][m], B as [n][k]).
__device__ __forceinline__ void lc_a_rows(uint32_t (&a)[4], const bf16* tile, int ld) {
    const int lane = threadIdx.x & 31;
    ldmatrix_x4(a, tile + (lane & 15) * ld + (lane >> 4) * 8);
}
__device__ __forceinline__ void lc_a_cols(uint32_t (&a)[4], const bf16* tile, int ld) {
    const int lane = threadIdx.x & 31;
    ldmatrix_x4_trans(a, tile + ((lane & 7) + ((lane >> 4) << 3)) * ld + ((lane >> 3) & 1) * 8);
}
__device__ __forceinline__ void lc_b_rows(uint32_t (&b)[4], const bf16* tile, int ld) {
    const int lane = threadIdx.x & 31;
    ldmatrix_x4_trans(b, tile + (lane & 15) * ld + (lane >> 4) * 8);
}
__device__ __forceinline__ void lc_b_cols(uint32_t (&b)[4], const bf16* tile, int ld) {
    const int lane = threadIdx.x & 31;
    ldmatrix_x4(b, tile + ((lane & 7) + ((lane >> 4) << 3)) * ld + ((lane >> 3) & 1) * 8);
}
// The 16x16 float32 tile of a warp's accumulators to and from shared memory.
__device__ __forceinline__ void lc_store(float* tile, int ld, const float (&acc)[2][4]) {
    const int g = (threadIdx.x & 31) >> 2, t = threadIdx.x & 3;
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
        *reinterpret_cast<float2*>(tile + g * ld + nb * 8 + 2 * t) = make_float2(acc[nb][0], acc[nb][1]);
        *reinterpret_cast<float2*>(tile + (g + 8) * ld + nb * 8 + 2 * t) = make_float2(acc[nb][2], acc[nb][3]);
    }
}
__device__ __forceinline__ void lc_load(float (&acc)[2][4], const float* tile, int ld) {
    const int g = (threadIdx.x & 31) >> 2, t = threadIdx.x & 3;
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
        const float2 lo = *reinterpret_cast<const float2*>(tile + g * ld + nb * 8 + 2 * t);
        const float2 hi = *reinterpret_cast<const float2*>(tile + (g + 8) * ld + nb * 8 + 2 * t);
        acc[nb][0] = lo.x, acc[nb][1] = lo.y, acc[nb][2] = hi.x, acc[nb][3] = hi.y;
    }
}

__device__ __forceinline__ void lc_split(float x, bf16& hi, bf16& lo) {
    hi = __float2bfloat16_rn(x);
    lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}
