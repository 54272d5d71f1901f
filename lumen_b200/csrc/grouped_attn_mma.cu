// Grouped-query attention of single rows (decode, short portions) over a bf16 cache on the warp-level tensor cores.
//
// A warp walks tiles of 16 cached rows with a running softmax of its own; the warps of a CTA are merged once at the end.  Cached rows
// are on the 16-row side of both products and up to 8 query heads of their key head on the 8-column side:
//   scores [16 rows, 8 heads] = K q^T: a lane's 16-byte load of a row serves two MMAs; the order of the contraction is free as long
//                               as q is held in the same order
//   O^T [values, 8 heads] += V^T P^T: a lane loads 16 bytes (8 values) of four rows; bytes of two rows are paired into the operands
//                               of one MMA per value of the eight, P^T comes from the scores by 8 x 8 transposes
// so that no tile passes through shared memory.  The weights P enter as a bf16 hi + lo pair.
#include <algorithm>

#include "grouped_attention.cuh"
#include "mma_common.cuh"
#include "tc_common.cuh"

namespace lumen {
namespace {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;
constexpr int kTileRows = 16, kStep = kWarps * kTileRows;

// KB: blocks of 32 numbers of a key; VB: blocks of 64 numbers of a value.
// grid (pieces, G * groups of kMmaHeads query heads, rows)
template <int KB, int VB>
__global__ void __launch_bounds__(kThreads, 1) grouped_mma_kernel(const GroupedArgs a, int append) {
    extern __shared__ __align__(16) float smem[];
    const int dim = (int)a.dim, vdim = (int)a.vdim, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    float *buf = smem + warp * dim;                                              // [warps][dim]
    float *wm = smem + kWarps * dim, *wl = wm + kWarps * kMmaHeads;              // [warps][heads]
    float *wctx = wl + kWarps * kMmaHeads;                                       // [warps][heads][vdim]
    __shared__ __align__(16) __nv_bfloat16 qs[kMmaHeads][KB * 32];
    const int R = (int)(a.H / a.G), groups = (R + kMmaHeads - 1) / kMmaHeads, hk = (int)blockIdx.y / groups, first = ((int)blockIdx.y % groups) * kMmaHeads;
    const int heads = min(kMmaHeads, R - first), h0 = hk * R + first;
    const float scale2 = a.scale * 1.4426950408889634f;  // weights are powers of two: exp(s scale - m) = 2^(s scale log2(e) - m')
    pdl_launch();
    bool ahead = append;  // (the cached rows of a layer that appends are older than this step, see grouped_rows_kernel)
    if (!ahead) pdl_wait();
    for (size_t m = blockIdx.z; m < a.B * a.S; m += gridDim.z) {
        const size_t b = m / a.S;
        const int pos = *a.d_len + (int)(m - b * a.S), lo = chunk_start(pos, a.chunk), len = pos + 1 - lo;
        const int per = piece_rows(len, a.nsplit), j0 = lo + (int)blockIdx.x * per, j1 = min(pos + 1, j0 + per);
        if (j0 >= j1) {  // (the same for the whole CTA)
            if (ahead) pdl_wait();
            ahead = false;
            continue;
        }
        __nv_bfloat16 *kbase = static_cast<__nv_bfloat16 *>(a.k) + (b * a.G + hk) * a.max_seq * dim;
        __nv_bfloat16 *vbase = static_cast<__nv_bfloat16 *>(a.v) + (b * a.G + hk) * a.max_seq * vdim;
        const float *u = a.u + m * a.u_ld;
        uint4 kr[KB][2], vr[4][VB];
        auto load_k = [&](int jb) {  // rows jb + g and jb + g + 8 (inside the piece: masked below)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const __nv_bfloat16 *row = kbase + (size_t)min(jb + g + 8 * i, j1 - 1) * dim;
#pragma unroll
                for (int kb = 0; kb < KB; ++kb) {
                    const int e = kb * 32 + 8 * t;
                    kr[kb][i] = e < dim ? __ldcg(reinterpret_cast<const uint4 *>(row + e)) : make_uint4(0u, 0u, 0u, 0u);
                }
            }
        };
        auto load_v = [&](int jb) {  // rows jb + 2t, 2t + 1, 2t + 8, 2t + 9
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const __nv_bfloat16 *row = vbase + (size_t)min(jb + 2 * t + (i & 1) + 8 * (i >> 1), j1 - 1) * vdim;
#pragma unroll
                for (int vb = 0; vb < VB; ++vb) {
                    const int e = vb * 64 + 8 * g;
                    vr[i][vb] = e < vdim ? __ldcg(reinterpret_cast<const uint4 *>(row + e)) : make_uint4(0u, 0u, 0u, 0u);
                }
            }
        };
        int jb = j0 + warp * kTileRows;
        const bool early = ahead && jb + kTileRows <= pos && jb < j1;  // nothing of the tile is appended by this step
        if (early) load_k(jb);
        if (ahead) pdl_wait();
        ahead = false;
        const size_t half = a.rot_dims / 2;
        const float *cos_row = a.cos_t + pos * half, *sin_row = a.sin_t + pos * half;
        if (warp < heads) head_norm_rotate(buf, u + (size_t)(h0 + warp) * dim, dim, a.q_gain, a.eps, (int)a.rot_dims, cos_row, sin_row, lane);
        for (int e = lane; e < KB * 32; e += 32) qs[warp][e] = __float2bfloat16_rn(warp < heads && e < dim ? buf[e] : 0.f);
        if (append && j1 == pos + 1 && warp == kWarps - 1) {
            // every group of query heads writes the row that it reads below (the same numbers)
            __syncwarp();
            head_norm_rotate(buf, u + a.u_k + (size_t)hk * dim, dim, a.k_gain, a.eps, (int)a.rot_dims, cos_row, sin_row, lane);
            for (int e = lane; e < dim; e += 32) kbase[(size_t)pos * dim + e] = __float2bfloat16_rn(buf[e]);
            for (int e = lane; e < vdim; e += 32) vbase[(size_t)pos * vdim + e] = __float2bfloat16_rn(u[a.u_v + (size_t)hk * vdim + e]);
        }
        __syncthreads();
        if (!early && jb < j1) load_k(jb);
        uint4 q[KB];
#pragma unroll
        for (int kb = 0; kb < KB; ++kb) q[kb] = *reinterpret_cast<const uint4 *>(&qs[g][kb * 32 + 8 * t]);
        float o[8][4];  // value 8 g + e (and 64 + 8 g + e) of heads 2t, 2t + 1
#pragma unroll
        for (int e = 0; e < 8; ++e)
#pragma unroll
            for (int c = 0; c < 4; ++c) o[e][c] = 0.f;
        float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};  // of heads 2t, 2t + 1; the sums are this lane's share
#pragma unroll 1
        for (; jb < j1; jb += kStep) {
            load_v(jb);
            float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int kb = 0; kb < KB; ++kb) {
                const uint32_t a0[4] = {kr[kb][0].x, kr[kb][1].x, kr[kb][0].y, kr[kb][1].y}, a1[4] = {kr[kb][0].z, kr[kb][1].z, kr[kb][0].w, kr[kb][1].w};
                mma16816(s, a0, q[kb].x, q[kb].y);
                mma16816(s, a1, q[kb].z, q[kb].w);
            }
            if (jb + kStep < j1) load_k(jb + kStep);
            const bool in0 = jb + g < j1, in1 = jb + g + 8 < j1;
            float r[2];
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                s[c] = in0 ? s[c] * scale2 : -INFINITY;
                s[2 + c] = in1 ? s[2 + c] * scale2 : -INFINITY;
                float mt = fmaxf(s[c], s[2 + c]);
#pragma unroll
                for (int d = 4; d < 32; d <<= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, d));
                mt = fmaxf(mt, mx[c]);  // finite: the tile's first row is inside the piece
                r[c] = tc::ex2(mx[c] - mt);
                mx[c] = mt;
                s[c] = tc::ex2(s[c] - mt);
                s[2 + c] = tc::ex2(s[2 + c] - mt);
                l[c] = fmaf(l[c], r[c], s[c] + s[2 + c]);
            }
            uint32_t ph[2], pl[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const uint32_t hi = tc::pack_bf16(s[2 * i], s[2 * i + 1]);
                ph[i] = transpose8x8(hi);
                pl[i] = transpose8x8(tc::pack_bf16(s[2 * i] - __uint_as_float(hi << 16), s[2 * i + 1] - __uint_as_float(hi & 0xffff0000u)));
            }
            if (__any_sync(0xffffffffu, r[0] != 1.f || r[1] != 1.f))
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    o[e][0] *= r[0]; o[e][1] *= r[1];
                    o[e][2] *= r[0]; o[e][3] *= r[1];
                }
            auto word = [](const uint4 &v, int i) { return i == 0 ? v.x : i == 1 ? v.y : i == 2 ? v.z : v.w; };
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const unsigned pick = e & 1 ? 0x7632 : 0x5410;  // the odd or the even number of two words
                uint32_t av[4] = {0u, 0u, 0u, 0u};
#pragma unroll
                for (int vb = 0; vb < VB; ++vb) {
                    av[vb] = __byte_perm(word(vr[0][vb], e / 2), word(vr[1][vb], e / 2), pick);
                    av[2 + vb] = __byte_perm(word(vr[2][vb], e / 2), word(vr[3][vb], e / 2), pick);
                }
                mma16816(o[e], av, ph[0], ph[1]);
                mma16816(o[e], av, pl[0], pl[1]);
            }
        }
#pragma unroll
        for (int c = 0; c < 2; ++c) {
#pragma unroll
            for (int d = 4; d < 32; d <<= 1) l[c] += __shfl_xor_sync(0xffffffffu, l[c], d);
            if (g == 0) {
                wm[warp * kMmaHeads + 2 * t + c] = mx[c];
                wl[warp * kMmaHeads + 2 * t + c] = l[c];
            }
#pragma unroll
            for (int e = 0; e < 8; ++e)
#pragma unroll
                for (int vb = 0; vb < VB; ++vb)
                    if (vb * 64 + 8 * g + e < vdim) wctx[(warp * kMmaHeads + 2 * t + c) * vdim + vb * 64 + 8 * g + e] = o[e][2 * vb + c];
        }
        __syncthreads();
        for (int i = tid; i < heads * vdim; i += kThreads) {
            const int hd = i / vdim, e = i - hd * vdim;
            float M = -INFINITY, L = 0.f, c = 0.f;
#pragma unroll
            for (int w = 0; w < kWarps; ++w) M = fmaxf(M, wm[w * kMmaHeads + hd]);
#pragma unroll
            for (int w = 0; w < kWarps; ++w) {
                const float f = tc::ex2(wm[w * kMmaHeads + hd] - M);  // (a warp without tiles: 2^-inf = 0)
                L = fmaf(wl[w * kMmaHeads + hd], f, L);
                c = fmaf(wctx[(w * kMmaHeads + hd) * vdim + e], f, c);
            }
            const size_t row = (m * a.H + h0 + hd) * a.nsplit + blockIdx.x;
            a.part_ctx[row * vdim + e] = c;
            if (e == 0) {
                a.part_ml[row * 2] = M * 0.6931471805599453f;
                a.part_ml[row * 2 + 1] = L;
            }
        }
        __syncthreads();
    }
}

template <int KB, int VB>
int launch(lumen_ctx *ctx, const GroupedArgs &a, bool append, cudaStream_t s) {
    const size_t smem = (kWarps * a.dim + 2 * kWarps * kMmaHeads + (size_t)kWarps * kMmaHeads * a.vdim) * sizeof(float);
    if (smem > 40 * 1024) LUMEN_CUDA(ctx, cudaFuncSetAttribute(grouped_mma_kernel<KB, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const size_t r = a.H / a.G, groups = (r + kMmaHeads - 1) / kMmaHeads;
    const dim3 grid((unsigned)a.nsplit, (unsigned)(a.G * groups), (unsigned)std::min<size_t>(a.B * a.S, 65535));
    return launch_pdl(ctx, grouped_mma_kernel<KB, VB>, grid, kThreads, smem, s, a, append ? 1 : 0);
}

}  // namespace

// Heads of at most 128 numbers in whole 16-byte pieces.
bool grouped_mma_usable(const GroupedArgs &a) {
    return a.dt == LUMEN_BF16 && a.dim <= 128 && a.vdim <= 128 && a.dim % 8 == 0 && a.vdim % 8 == 0;
}

int launch_grouped_mma(lumen_ctx *ctx, const GroupedArgs &a, bool append, cudaStream_t s) {
    const bool wide = a.vdim > 64;
    switch ((a.dim + 31) / 32) {
        case 1: return wide ? launch<1, 2>(ctx, a, append, s) : launch<1, 1>(ctx, a, append, s);
        case 2: return wide ? launch<2, 2>(ctx, a, append, s) : launch<2, 1>(ctx, a, append, s);
        case 3: return wide ? launch<3, 2>(ctx, a, append, s) : launch<3, 1>(ctx, a, append, s);
        default: return wide ? launch<4, 2>(ctx, a, append, s) : launch<4, 1>(ctx, a, append, s);
    }
}

}  // namespace lumen
