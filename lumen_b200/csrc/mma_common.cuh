// Warp-level bf16 MMA (m16n8k16, f32 accumulators) for steps of few query rows, where a tcgen05 tile of 128 rows would be nearly
// empty.  With g = lane / 4 and t = lane % 4: a[0], a[2] hold row g, columns 2t, 2t + 1 and 2t + 8, 2t + 9; a[1], a[3] row g + 8;
// b0, b1 rows 2t, 2t + 1 and 2t + 8, 2t + 9 of column g; d[0], d[1] row g, columns 2t, 2t + 1; d[2], d[3] row g + 8.
#pragma once

#include "common.cuh"

namespace lumen {

__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Transpose of an 8 x 8 matrix of 16-bit numbers whose row g, columns 2t, 2t + 1 this lane holds.
__device__ __forceinline__ uint32_t transpose8x8(uint32_t x) {
    uint32_t y;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
    return y;
}

}  // namespace lumen
