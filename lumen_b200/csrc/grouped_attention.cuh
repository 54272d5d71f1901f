// What the kernels of grouped-query attention over chunks share.
#pragma once

#include "attn_decode.cuh"
#include "decoder_kernels.cuh"

namespace lumen {

constexpr int kPiece = 32;     // pieces of a row's context start at multiples of this many rows from the chunk's start
constexpr int kMmaHeads = 8;   // query heads a CTA of the MMA kernel takes

// The one-row kernel on the tensor cores (bf16 cache): one CTA per (piece, key head and up to kMmaHeads of its query heads, row).
bool grouped_mma_usable(const GroupedArgs &a);
int launch_grouped_mma(lumen_ctx *ctx, const GroupedArgs &a, bool append, cudaStream_t s);

__device__ __forceinline__ int chunk_start(int pos, size_t chunk) { return chunk ? (int)((size_t)pos / chunk * chunk) : 0; }
__device__ __forceinline__ int piece_rows(int len, int nsplit) { return ((len + nsplit - 1) / nsplit + kPiece - 1) / kPiece * kPiece; }

// One head vector by one warp: RMS norm with gains, then the pairs (i, i + rot_dims / 2) turn.  buf: shared memory [dim].
__device__ __forceinline__ void head_norm_rotate(float *buf, const float *src, int dim, const float *gain, float eps, int rot_dims,
                                                 const float *cos_row, const float *sin_row, int lane) {
    float ss = 0.f;
#pragma unroll 4
    for (int i = lane; i < dim; i += 32) {
        const float v = src[i];
        buf[i] = v;
        ss = fmaf(v, v, ss);
    }
    ss = attn_warp_sum(ss);
    const float inv = __fdiv_rn(1.0f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)dim), eps)));
    for (int i = lane; i < dim; i += 32) buf[i] = __fmul_rn(__fmul_rn(buf[i], inv), gain[i]);
    __syncwarp();
    const int half = rot_dims / 2;
    for (int i = lane; i < half; i += 32) {
        const float x = buf[i], y = buf[i + half], c = cos_row[i], s = sin_row[i];
        buf[i] = __fsub_rn(__fmul_rn(x, c), __fmul_rn(y, s));
        buf[i + half] = __fadd_rn(__fmul_rn(y, c), __fmul_rn(x, s));
    }
    __syncwarp();
}

}  // namespace lumen
