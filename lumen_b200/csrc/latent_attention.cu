// Latent attention: keys and values of all heads come from one normed latent per token, plus one rotated key part that the
// heads share; the cache holds these two (a row: latent, rotated part, zeros up to the pitch).
//
// With W_uk moved to the query side a head's score against row j is q_lat . c_j + q_rot . k_rot_j with q_lat = W_uk^T q, and
// its output is W_uv (sum_j p_j c_j): the cached rows serve as keys and as values for every head and nothing is expanded.
//   latent_append_kernel  norm, rotation, cache rows of the step
//   latent_absorb_kernel  q_lat and the rotated query part (and, in decode steps, the append in the same launch)
//   latent_scores_kernel  scores, running softmax and weighted latents in 32-bit FMAs, any sizes; f32 models, and
//                         sizes that the tensor-core kernels (latent_attn_mma.cu, attn_prefill_tc.cu) do not take
//   latent_value_kernel   pieces of the context merged, W_uv, output gate
#include <algorithm>

#include "decoder_kernels.cuh"
#include "gemv_rows.cuh"

namespace lumen {
namespace {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;

// Rotates the interleaved pair of elements (i, i ^ 1) of a vector of which the first rot_dims elements turn.
__device__ __forceinline__ float rotated(const float *v, size_t i, size_t rot_dims, const float *cos_row, const float *sin_row) {
    if (i >= rot_dims) return v[i];
    const float c = cos_row[i >> 1], s = sin_row[i >> 1];
    const float x = v[i & ~(size_t)1], y = v[i | 1];
    return (i & 1) ? __fadd_rn(__fmul_rn(y, c), __fmul_rn(x, s)) : __fsub_rn(__fmul_rn(x, c), __fmul_rn(y, s));
}

// NT threads (a warp, or the whole CTA) share a row.
template <typename T, int NT>
__device__ __forceinline__ void append_row(const LatentArgs &a, size_t m, float *red, int tid) {
    const size_t b = m / a.S, pos = (size_t)*a.d_len + (m - b * a.S);
    const float *d = a.u + m * a.u_ld + a.u_kv;
    T *row = static_cast<T *>(a.cache) + (b * a.max_seq + pos) * a.pitch;
    float ss = 0.f;
#pragma unroll (NT == 32 ? 16 : 4)
    for (size_t i = tid; i < a.rank; i += NT) ss = fmaf(d[i], d[i], ss);
    ss = warp_sum(ss);
    if (NT > 32) {
        if ((tid & 31) == 0) red[tid >> 5] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int w = 0; w < NT / 32; ++w) ss += red[w];
    }
    const float inv = __fdiv_rn(1.0f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)a.rank), a.eps)));
    const size_t half = a.rot_dims / 2;
#pragma unroll (NT == 32 ? 16 : 4)
    for (size_t i = tid; i < a.rank; i += NT) row[i] = from_f32<T>(__fmul_rn(__fmul_rn(d[i], inv), a.latent_gain[i]));
    for (size_t i = a.rank + tid; i < a.pitch; i += NT) {
        float v = 0.f;
        if (i < a.rank + a.rot_dim) v = rotated(d + a.rank, i - a.rank, a.rot_dims, a.cos_t + pos * half, a.sin_t + pos * half);
        row[i] = from_f32<T>(v);
    }
}

template <typename T>
__global__ void __launch_bounds__(kThreads) latent_append_kernel(const LatentArgs a) {
    const size_t m = (size_t)blockIdx.x * kWarps + (threadIdx.x >> 5);  // one warp per row
    if (m < a.B * a.S) append_row<T, 32>(a, m, nullptr, threadIdx.x & 31);
}

// grid (heads, chunks of 64 latent columns (+ 1 when the first head's CTA there appends the cache row), rows)
constexpr int kAbsorbCols = 64, kColGroups = kAbsorbCols / 8, kSlices = kThreads / kColGroups;
template <typename T>
__global__ void __launch_bounds__(kThreads) latent_absorb_kernel(const LatentArgs a, int chunks) {
    __shared__ float part[kSlices][kAbsorbCols];
    const int tid = threadIdx.x;
    const size_t h = blockIdx.x, m = blockIdx.z;
    // the first weight vectors of this thread are requested while the projections still run
    constexpr int kQ = sizeof(T) / 2;
    const int cg = tid % kColGroups, slice = tid / kColGroups;
    const size_t r0 = (size_t)blockIdx.y * kAbsorbCols + cg * 8;
    const T *w = static_cast<const T *>(a.wuk) + h * a.dim * a.rank + r0;
    const bool vec = a.rank % 8 == 0, mine = (int)blockIdx.y < chunks && r0 < a.rank;
    uint4 pre[kAhead][kQ];
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
        if (vec && mine && slice + i * kSlices < a.dim)
#pragma unroll
            for (int k = 0; k < kQ; ++k) pre[i][k] = ld_stream_u4(reinterpret_cast<const uint4 *>(w + (slice + i * kSlices) * a.rank) + k);
    pdl_launch();
    pdl_wait();
    if ((int)blockIdx.y == chunks) {
        if (h == 0) append_row<T, kThreads>(a, m, &part[0][0], tid);
        return;
    }
    const float *q = a.u + m * a.u_ld + h * (a.dim + a.rot_dim);
    T *out = static_cast<T *>(a.qf) + (m * a.H + h) * a.pitch;
    if (blockIdx.y == 0) {  // rotated part and the zeros behind it
        const size_t pos = (size_t)*a.d_len + m % a.S, half = a.rot_dims / 2;
        for (size_t i = a.rank + tid; i < a.pitch; i += kThreads)
            out[i] = from_f32<T>(i < a.rank + a.rot_dim ? rotated(q + a.dim, i - a.rank, a.rot_dims, a.cos_t + pos * half, a.sin_t + pos * half) : 0.f);
    }
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    if (vec) {
        auto add = [&](const uint4 (&v)[kQ], float x) {
            if constexpr (sizeof(T) == 4) {
#pragma unroll
                for (int k = 0; k < kQ; ++k) {
                    acc[4 * k] = fmaf(__uint_as_float(v[k].x), x, acc[4 * k]); acc[4 * k + 1] = fmaf(__uint_as_float(v[k].y), x, acc[4 * k + 1]);
                    acc[4 * k + 2] = fmaf(__uint_as_float(v[k].z), x, acc[4 * k + 2]); acc[4 * k + 3] = fmaf(__uint_as_float(v[k].w), x, acc[4 * k + 3]);
                }
            } else {
                acc[0] = fmaf(bf16_lo(v[0].x), x, acc[0]); acc[1] = fmaf(bf16_hi(v[0].x), x, acc[1]);
                acc[2] = fmaf(bf16_lo(v[0].y), x, acc[2]); acc[3] = fmaf(bf16_hi(v[0].y), x, acc[3]);
                acc[4] = fmaf(bf16_lo(v[0].z), x, acc[4]); acc[5] = fmaf(bf16_hi(v[0].z), x, acc[5]);
                acc[6] = fmaf(bf16_lo(v[0].w), x, acc[6]); acc[7] = fmaf(bf16_hi(v[0].w), x, acc[7]);
            }
        };
        if (mine) {
#pragma unroll
            for (int i = 0; i < kAhead; ++i)
                if (slice + i * kSlices < a.dim) add(pre[i], q[slice + i * kSlices]);
            for (size_t d = slice + kAhead * kSlices; d < a.dim; d += kSlices) {
                uint4 v[kQ];
#pragma unroll
                for (int k = 0; k < kQ; ++k) v[k] = ld_stream_u4(reinterpret_cast<const uint4 *>(w + d * a.rank) + k);
                add(v, q[d]);
            }
        }
    } else {
        for (size_t d = slice; d < a.dim; d += kSlices) {
            const float x = q[d];
#pragma unroll
            for (int j = 0; j < 8; ++j)
                if (r0 + j < a.rank) acc[j] = fmaf(to_f32(w[d * a.rank + j]), x, acc[j]);
        }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) part[slice][cg * 8 + j] = acc[j];
    __syncthreads();
    if (tid < kAbsorbCols) {
        const size_t r = (size_t)blockIdx.y * kAbsorbCols + tid;
        float v = 0.f;
#pragma unroll
        for (int s = 0; s < kSlices; ++s) v += part[s][tid];
        if (r < a.rank) out[r] = from_f32<T>(v);
    }
}

// grid (splits, query rows m * H + h): 4 warps share the rows of the split, each with a running softmax; merged at the end.
// A lane holds elements lane + 32 i of the latent.
constexpr int kScoreWarps = 4;
template <typename T, int NI>
__global__ void __launch_bounds__(kScoreWarps * 32) latent_scores_kernel(const LatentArgs a) {
    extern __shared__ float smem[];
    float *q = smem;                        // [rank + rot_dim]
    float *wctx = q + a.rank + a.rot_dim;   // [warps][rank]
    __shared__ float wm[kScoreWarps], wl[kScoreWarps];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int rank = (int)a.rank, width = (int)(a.rank + a.rot_dim);
    pdl_wait();
    pdl_launch();
    for (size_t row = blockIdx.y; row < a.B * a.S * a.H; row += gridDim.y) {
        const size_t m = row / a.H, b = m / a.S, past = (size_t)*a.d_len, total = past + a.S;
        const size_t seen = past + (m - b * a.S) + 1;
        const int pieces = latent_pieces((int)total, a.nsplit);
        if ((int)blockIdx.x >= pieces) return;
        const size_t j0 = latent_piece_start((int)total, pieces, blockIdx.x), j1 = min(seen, (size_t)latent_piece_start((int)total, pieces, blockIdx.x + 1));
        const T *qsrc = static_cast<const T *>(a.qf) + row * a.pitch;
        __syncthreads();
        for (int i = tid; i < width; i += kScoreWarps * 32) q[i] = to_f32(qsrc[i]);
        __syncthreads();
        const T *cache = static_cast<const T *>(a.cache) + b * a.max_seq * a.pitch;
        float ctx[NI], mx = -INFINITY, l = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) ctx[i] = 0.f;
        for (size_t j = j0 + warp; j < j1; j += kScoreWarps) {
            const T *c = cache + j * a.pitch;
            float cv[NI], s = 0.f;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int e = lane + 32 * i;
                cv[i] = e < rank ? to_f32(c[e]) : 0.f;
            }
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int e = lane + 32 * i;
                if (e < rank) s = fmaf(q[e], cv[i], s);
            }
            for (int e = rank + lane; e < width; e += 32) s = fmaf(q[e], to_f32(c[e]), s);
            s = warp_sum(s) * a.scale;
            const float mn = fmaxf(mx, s), r = expf(mx - mn), p = expf(s - mn);
            mx = mn;
            l = fmaf(l, r, p);
#pragma unroll
            for (int i = 0; i < NI; ++i) ctx[i] = fmaf(ctx[i], r, p * cv[i]);
        }
        if (lane == 0) {
            wm[warp] = mx;
            wl[warp] = l;
        }
#pragma unroll
        for (int i = 0; i < NI; ++i)
            if (lane + 32 * i < rank) wctx[warp * rank + lane + 32 * i] = ctx[i];
        __syncthreads();
        float M = wm[0];
#pragma unroll
        for (int w = 1; w < kScoreWarps; ++w) M = fmaxf(M, wm[w]);
        float f[kScoreWarps], lsum = 0.f;
#pragma unroll
        for (int w = 0; w < kScoreWarps; ++w) {
            f[w] = wm[w] == -INFINITY ? 0.f : expf(wm[w] - M);
            lsum = fmaf(wl[w], f[w], lsum);
        }
        const size_t o = row * a.nsplit + blockIdx.x;
        for (int e = tid; e < rank; e += kScoreWarps * 32) {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < kScoreWarps; ++w) v = fmaf(wctx[w * rank + e], f[w], v);
            a.part_ctx[o * rank + e] = v;
        }
        if (tid == 0) {
            a.part_ml[o * 2] = M;
            a.part_ml[o * 2 + 1] = lsum;
        }
    }
}

// grid (heads, chunks of value rows, rows)
constexpr int kValueRows = 16, kValueThreads = 512, kValueGroups = kValueThreads / 128;
template <typename T>
__global__ void __launch_bounds__(kValueThreads) latent_value_kernel(const LatentArgs a) {
    extern __shared__ __align__(16) float smem[];
    const size_t rank4 = (a.rank + 3) & ~(size_t)3;
    float *ctx = smem;                        // [groups][rank4]: shares of the pieces, summed into the first
    float *f = ctx + kValueGroups * rank4;    // [nsplit]
    __shared__ float inv_s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const size_t h = blockIdx.x, m = blockIdx.z, o = (m * a.H + h) * a.nsplit;
    constexpr int VEC = 16 / sizeof(T);
    const bool vec_ok = a.rank % VEC == 0;
    const size_t v0 = (size_t)blockIdx.y * kValueRows + warp, v1 = min(a.vdim, (size_t)(blockIdx.y + 1) * kValueRows);
    const T *w = static_cast<const T *>(a.wuv) + h * a.vdim * a.rank;
    uint4 pre[kAhead];
    const int nv = (int)(a.rank / VEC);
    if (vec_ok && v0 < v1) row_ahead(reinterpret_cast<const uint4 *>(w + v0 * a.rank), nv, lane, pre);
    pdl_launch();
    pdl_wait();
    const int pieces = latent_pieces(*a.d_len + (int)a.S, a.nsplit);
    if (warp == 0) {
        float M = -INFINITY;
        for (int s = lane; s < pieces; s += 32) M = fmaxf(M, a.part_ml[(o + s) * 2]);
#pragma unroll
        for (int k = 16; k > 0; k >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, k));
        float l = 0.f;
        for (int s = lane; s < pieces; s += 32) {
            const float ms = a.part_ml[(o + s) * 2], w = ms == -INFINITY ? 0.f : expf(ms - M);
            f[s] = w;
            l = fmaf(a.part_ml[(o + s) * 2 + 1], w, l);
        }
        l = warp_sum(l);
        if (lane == 0) inv_s = __fdiv_rn(1.0f, l);
    }
    __syncthreads();
    const float inv = inv_s;
    if (a.rank % 4 == 0) {  // groups of 128 threads, each with every fourth piece; a thread owns four adjacent columns
        const int group = tid >> 7;
        for (size_t c = tid & 127; c < a.rank / 4; c += 128) {
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
            for (int s = group; s < pieces; s += kValueGroups) {
                const float4 p = reinterpret_cast<const float4 *>(a.part_ctx + (o + s) * a.rank)[c];
                const float w = f[s];
                v.x = fmaf(p.x, w, v.x); v.y = fmaf(p.y, w, v.y); v.z = fmaf(p.z, w, v.z); v.w = fmaf(p.w, w, v.w);
            }
            reinterpret_cast<float4 *>(ctx + group * rank4)[c] = make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv);
        }
        __syncthreads();
        for (size_t r = tid; r < a.rank; r += kValueThreads) {
            float v = ctx[r];
#pragma unroll
            for (int g = 1; g < kValueGroups; ++g) v += ctx[g * rank4 + r];
            ctx[r] = v;
        }
    } else {
        for (size_t r = tid; r < a.rank; r += kValueThreads) {
            float v = 0.f;
            for (int s = 0; s < pieces; ++s) v = fmaf(a.part_ctx[(o + s) * a.rank + r], f[s], v);
            ctx[r] = v * inv;
        }
    }
    __syncthreads();
    const float gate = sigmoid_f(a.u[m * a.u_ld + a.u_gate + h]);
    for (size_t v = v0; v < v1; v += kValueThreads / 32) {
        float d;
        if (vec_ok) {
            const uint4 *wrow = reinterpret_cast<const uint4 *>(w + v * a.rank);
            if (v != v0) batch_load(wrow, 0, nv, lane, pre);
            d = row_dot_ahead<T>(wrow, ctx, nv, lane, pre);
        } else {
            d = row_dot_scalar<T>(w + v * a.rank, ctx, (int)a.rank, lane);
        }
        const float y = warp_sum(d) * gate;
        if (lane == 0) {
            const size_t at = (m * a.H + h) * a.vdim + v;
            if (a.out) a.out[at] = y;
            if (a.out_hi) store_split(y, a.out_hi, a.out_lo, at);
        }
    }
}

template <typename T>
int launch_scores_t(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s) {
    const size_t smem = ((1 + kScoreWarps) * a.rank + a.rot_dim) * sizeof(float);
    const dim3 grid((unsigned)a.nsplit, (unsigned)std::min<size_t>(65535, a.B * a.S * a.H));
#define LUMEN_SCORES(NI_)                                                                                                                \
    do {                                                                                                                                 \
        if (smem > 48 * 1024) LUMEN_CUDA(ctx, cudaFuncSetAttribute(latent_scores_kernel<T, NI_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        return launch_pdl(ctx, latent_scores_kernel<T, NI_>, grid, kScoreWarps * 32, smem, s, a);                                         \
    } while (0)
    if (a.rank <= 128) LUMEN_SCORES(4);
    if (a.rank <= 512) LUMEN_SCORES(16);
    LUMEN_SCORES(32);
#undef LUMEN_SCORES
}

}  // namespace

int launch_latent_append(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s) {
    if (a.dt == LUMEN_F32) latent_append_kernel<float><<<(unsigned)((a.B * a.S + kWarps - 1) / kWarps), kThreads, 0, s>>>(a);
    else latent_append_kernel<__nv_bfloat16><<<(unsigned)((a.B * a.S + kWarps - 1) / kWarps), kThreads, 0, s>>>(a);
    LUMEN_LAUNCHED(ctx);
    return LUMEN_OK;
}

int launch_latent_absorb(lumen_ctx *ctx, const LatentArgs &a, bool append, cudaStream_t s) {
    const size_t rows = a.B * a.S;
    if (rows > 65535) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "latent attention: %zu rows in one step", rows);
    const int chunks = (int)((a.rank + kAbsorbCols - 1) / kAbsorbCols);
    const dim3 grid((unsigned)a.H, (unsigned)(chunks + (append ? 1 : 0)), (unsigned)rows);
    return launch_pdl(ctx, a.dt == LUMEN_F32 ? latent_absorb_kernel<float> : latent_absorb_kernel<__nv_bfloat16>, grid, kThreads, 0, s, a, chunks);
}

int launch_latent_scores(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s) {
    if (a.rank > 1024) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "latent of %zu numbers (at most 1024)", a.rank);
    return a.dt == LUMEN_F32 ? launch_scores_t<float>(ctx, a, s) : launch_scores_t<__nv_bfloat16>(ctx, a, s);
}

int launch_latent_value(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s) {
    const size_t rows = a.B * a.S;
    if (rows > 65535) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "latent attention: %zu rows in one step", rows);
    const size_t smem = (kValueGroups * ((a.rank + 3) & ~(size_t)3) + a.nsplit) * sizeof(float);
    const dim3 grid((unsigned)a.H, (unsigned)((a.vdim + kValueRows - 1) / kValueRows), (unsigned)rows);
    return launch_pdl(ctx, a.dt == LUMEN_F32 ? latent_value_kernel<float> : latent_value_kernel<__nv_bfloat16>, grid, kValueThreads, smem, s, a);
}

}  // namespace lumen
