// Device helpers of the streaming vector-matrix kernels (gemv.cu, moe.cu): dot products of weight rows read once from
// HBM with 128-bit streaming loads against vectors staged in shared memory, one warp per row (or group of rows).
#pragma once

#include "common.cuh"

namespace lumen {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

__device__ __forceinline__ float4 ld_stream_f4(const float4 *p) { return __ldcs(p); }
__device__ __forceinline__ uint4 ld_stream_u4(const uint4 *p) { return __ldcs(p); }

__device__ __forceinline__ float bf16_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }

// Accumulate one row (`wrow`, K elements) against MB staged vectors.  Vector path needs K % VEC == 0
// and a 16-byte aligned row; otherwise the scalar path runs.
template <typename WT, int MB>
__device__ __forceinline__ void row_dot(const WT *__restrict__ wrow, const float *xs, size_t K, int lane, bool vec_ok,
                                        float (&acc)[MB]) {
    constexpr int kUnroll = 8;
    if constexpr (sizeof(WT) == 4) {
        if (vec_ok) {
            const float4 *w4 = reinterpret_cast<const float4 *>(wrow);
            const size_t n4 = K / 4;
            for (size_t base = 0; base < n4; base += 32 * kUnroll) {
                float4 wv[kUnroll];
#pragma unroll
                for (int u = 0; u < kUnroll; ++u) {
                    size_t i = base + (size_t)u * 32 + lane;
                    wv[u] = (i < n4) ? ld_stream_f4(w4 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
                }
#pragma unroll
                for (int u = 0; u < kUnroll; ++u) {
                    size_t i = base + (size_t)u * 32 + lane;
                    if (i < n4) {
#pragma unroll
                        for (int m = 0; m < MB; ++m) {
                            float4 xv = *reinterpret_cast<const float4 *>(xs + (size_t)m * K + i * 4);
                            acc[m] = fmaf(wv[u].x, xv.x, acc[m]);
                            acc[m] = fmaf(wv[u].y, xv.y, acc[m]);
                            acc[m] = fmaf(wv[u].z, xv.z, acc[m]);
                            acc[m] = fmaf(wv[u].w, xv.w, acc[m]);
                        }
                    }
                }
            }
            return;
        }
        for (size_t k = lane; k < K; k += 32) {
            float w = reinterpret_cast<const float *>(wrow)[k];
#pragma unroll
            for (int m = 0; m < MB; ++m) acc[m] = fmaf(w, xs[(size_t)m * K + k], acc[m]);
        }
    } else {
        if (vec_ok) {
            const uint4 *w8 = reinterpret_cast<const uint4 *>(wrow);
            const size_t n8 = K / 8;
            for (size_t base = 0; base < n8; base += 32 * kUnroll) {
                uint4 wv[kUnroll];
#pragma unroll
                for (int u = 0; u < kUnroll; ++u) {
                    size_t i = base + (size_t)u * 32 + lane;
                    wv[u] = (i < n8) ? ld_stream_u4(w8 + i) : make_uint4(0u, 0u, 0u, 0u);
                }
#pragma unroll
                for (int u = 0; u < kUnroll; ++u) {
                    size_t i = base + (size_t)u * 32 + lane;
                    if (i < n8) {
#pragma unroll
                        for (int m = 0; m < MB; ++m) {
                            const float4 *xp = reinterpret_cast<const float4 *>(xs + (size_t)m * K + i * 8);
                            float4 x0 = xp[0], x1 = xp[1];
                            acc[m] = fmaf(bf16_lo(wv[u].x), x0.x, acc[m]);
                            acc[m] = fmaf(bf16_hi(wv[u].x), x0.y, acc[m]);
                            acc[m] = fmaf(bf16_lo(wv[u].y), x0.z, acc[m]);
                            acc[m] = fmaf(bf16_hi(wv[u].y), x0.w, acc[m]);
                            acc[m] = fmaf(bf16_lo(wv[u].z), x1.x, acc[m]);
                            acc[m] = fmaf(bf16_hi(wv[u].z), x1.y, acc[m]);
                            acc[m] = fmaf(bf16_lo(wv[u].w), x1.z, acc[m]);
                            acc[m] = fmaf(bf16_hi(wv[u].w), x1.w, acc[m]);
                        }
                    }
                }
            }
            return;
        }
        for (size_t k = lane; k < K; k += 32) {
            float w = __bfloat162float(reinterpret_cast<const __nv_bfloat16 *>(wrow)[k]);
#pragma unroll
            for (int m = 0; m < MB; ++m) acc[m] = fmaf(w, xs[(size_t)m * K + k], acc[m]);
        }
    }
}

// A row in batches of kAhead x 32 vectors with the next batch always in flight.  The first batch is requested ahead of time (while
// an earlier kernel still runs) and the next few KB of the row handed to the L2 (not more: all rows of a large matrix at once
// would push one another out).  n: vectors of the row.
constexpr int kAhead = 4;  // (registers: more would reduce the CTAs an SM holds)
__device__ __forceinline__ void batch_load(const uint4 *__restrict__ row, int base, int n, int lane, uint4 (&v)[kAhead]) {
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
        const int i = base + u * 32 + lane;
        v[u] = i < n ? ld_stream_u4(row + i) : make_uint4(0u, 0u, 0u, 0u);
    }
}
__device__ __forceinline__ void row_ahead(const uint4 *__restrict__ row, int n, int lane, uint4 (&pre)[kAhead]) {
    batch_load(row, 0, n, lane, pre);
#pragma unroll 1
    for (int i = kAhead * 32 + lane * 8; i < min(n, 512); i += 256) asm volatile("prefetch.global.L2 [%0];" ::"l"(row + i));
}
template <typename WT>
__device__ __forceinline__ float vec_dot(uint4 w, const float *x, float acc) {
    const float4 x0 = *reinterpret_cast<const float4 *>(x);
    if constexpr (sizeof(WT) == 4) {
        acc = fmaf(__uint_as_float(w.x), x0.x, acc);
        acc = fmaf(__uint_as_float(w.y), x0.y, acc);
        acc = fmaf(__uint_as_float(w.z), x0.z, acc);
        return fmaf(__uint_as_float(w.w), x0.w, acc);
    } else {
        const float4 x1 = *reinterpret_cast<const float4 *>(x + 4);
        acc = fmaf(bf16_lo(w.x), x0.x, acc);
        acc = fmaf(bf16_hi(w.x), x0.y, acc);
        acc = fmaf(bf16_lo(w.y), x0.z, acc);
        acc = fmaf(bf16_hi(w.y), x0.w, acc);
        acc = fmaf(bf16_lo(w.z), x1.x, acc);
        acc = fmaf(bf16_hi(w.z), x1.y, acc);
        acc = fmaf(bf16_lo(w.w), x1.z, acc);
        return fmaf(bf16_hi(w.w), x1.w, acc);
    }
}
template <typename WT>
__device__ __forceinline__ float row_dot_ahead(const uint4 *__restrict__ row, const float *xs, int n, int lane, uint4 (&cur)[kAhead],
                                               const uint4 *__restrict__ next_row = nullptr) {  // its first batch is left in cur
    constexpr int VEC = 16 / sizeof(WT);
    float acc = 0.f;
#pragma unroll 1
    for (int base = 0; base < n; base += kAhead * 32) {
        uint4 next[kAhead];
        if (next_row && base + kAhead * 32 >= n) batch_load(next_row, 0, n, lane, next);
        else batch_load(row, base + kAhead * 32, n, lane, next);
#pragma unroll
        for (int u = 0; u < kAhead; ++u) {
            const int i = base + u * 32 + lane;
            if (i < n) acc = vec_dot<WT>(cur[u], xs + i * VEC, acc);
        }
#pragma unroll
        for (int u = 0; u < kAhead; ++u) cur[u] = next[u];
    }
    return acc;
}
// Any row length and alignment.
template <typename WT>
__device__ __forceinline__ float row_dot_scalar(const WT *__restrict__ row, const float *xs, int K, int lane) {
    float acc = 0.f;
#pragma unroll 1
    for (int k = lane; k < K; k += 32) {
        float w;
        if constexpr (sizeof(WT) == 4) w = row[k];
        else w = __bfloat162float(row[k]);
        acc = fmaf(w, xs[k], acc);
    }
    return acc;
}

// RR rows of W against MB staged vectors at once: every 16 bytes of x read from shared memory feed RR rows, so
// the shared-memory traffic per weight byte is MB / RR instead of MB (with MB = 8 and one row at a time the
// kernel was bound by shared memory, not by HBM).  Vector path only (K % VEC == 0, 16-byte aligned rows).
template <typename WT, int MB, int RR>
__device__ __forceinline__ void rows_dot(const WT *const (&rows)[RR], const float *xs, size_t K, int lane, float (&acc)[RR][MB]) {
    constexpr int VEC = 16 / sizeof(WT);
    constexpr int kUnroll = 4;
    const size_t nv = K / VEC;
    for (size_t base = 0; base < nv; base += 32 * kUnroll) {
        uint4 wv[RR][kUnroll];
#pragma unroll
        for (int u = 0; u < kUnroll; ++u) {
            const size_t i = base + (size_t)u * 32 + lane;
#pragma unroll
            for (int r = 0; r < RR; ++r)
                wv[r][u] = (i < nv) ? ld_stream_u4(reinterpret_cast<const uint4 *>(rows[r]) + i) : make_uint4(0u, 0u, 0u, 0u);
        }
#pragma unroll
        for (int u = 0; u < kUnroll; ++u) {
            const size_t i = base + (size_t)u * 32 + lane;
            if (i < nv) {
#pragma unroll
                for (int m = 0; m < MB; ++m) {
                    const float4 *xp = reinterpret_cast<const float4 *>(xs + (size_t)m * K + i * VEC);
                    const float4 x0 = xp[0];
                    if constexpr (sizeof(WT) == 4) {
#pragma unroll
                        for (int r = 0; r < RR; ++r) {
                            acc[r][m] = fmaf(__uint_as_float(wv[r][u].x), x0.x, acc[r][m]);
                            acc[r][m] = fmaf(__uint_as_float(wv[r][u].y), x0.y, acc[r][m]);
                            acc[r][m] = fmaf(__uint_as_float(wv[r][u].z), x0.z, acc[r][m]);
                            acc[r][m] = fmaf(__uint_as_float(wv[r][u].w), x0.w, acc[r][m]);
                        }
                    } else {
                        const float4 x1 = xp[1];
#pragma unroll
                        for (int r = 0; r < RR; ++r) {
                            acc[r][m] = fmaf(bf16_lo(wv[r][u].x), x0.x, acc[r][m]);
                            acc[r][m] = fmaf(bf16_hi(wv[r][u].x), x0.y, acc[r][m]);
                            acc[r][m] = fmaf(bf16_lo(wv[r][u].y), x0.z, acc[r][m]);
                            acc[r][m] = fmaf(bf16_hi(wv[r][u].y), x0.w, acc[r][m]);
                            acc[r][m] = fmaf(bf16_lo(wv[r][u].z), x1.x, acc[r][m]);
                            acc[r][m] = fmaf(bf16_hi(wv[r][u].z), x1.y, acc[r][m]);
                            acc[r][m] = fmaf(bf16_lo(wv[r][u].w), x1.z, acc[r][m]);
                            acc[r][m] = fmaf(bf16_hi(wv[r][u].w), x1.w, acc[r][m]);
                        }
                    }
                }
            }
        }
    }
}

}  // namespace lumen
