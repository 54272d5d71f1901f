// Matrix-memory layers (the mLSTM of "xLSTM: Extended Long Short-Term Memory", Beck et al.), token by token.
//
// A head's memory S [dim, vdim], its normaliser n [dim] and its running maximum m live in 32-bit floats in the cache.  The
// columns of S are independent given the gates, so a cluster of up to 8 CTAs shares a head, each with a slice of the columns;
// only the sum of squares of the head's output (its RMS norm) crosses the cluster.  A thread owns the same elements
// of S from the first token of a portion to the last, and T tokens are applied per pass over S.
#include <algorithm>
#include <cooperative_groups.h>

#include "decoder_kernels.cuh"
#include "gemv_rows.cuh"
#include "mlstm_gates.cuh"

namespace lumen {
namespace {

namespace cg = cooperative_groups;

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;
constexpr int kPre = 16;  // rows of S a thread requests before it waits for the projections (decode)

template <int VEC>
struct Cols {
    float v[VEC];
};
template <int VEC>
__device__ __forceinline__ Cols<VEC> load_cols(const float *p) {
    Cols<VEC> c;
    if constexpr (VEC == 4) {
        const float4 f = *reinterpret_cast<const float4 *>(p);
        c.v[0] = f.x; c.v[1] = f.y; c.v[2] = f.z; c.v[3] = f.w;
    } else {
        c.v[0] = *p;
    }
    return c;
}
template <int VEC>
__device__ __forceinline__ void store_cols(float *p, const Cols<VEC> &c) {
    if constexpr (VEC == 4) *reinterpret_cast<float4 *>(p) = make_float4(c.v[0], c.v[1], c.v[2], c.v[3]);
    else *p = c.v[0];
}

// grid (slices of the columns = cluster, heads, batch); cols = columns per CTA, nx = cols / VEC threads across, ny groups of rows
template <int VEC, int T>
__global__ void __launch_bounds__(kThreads) mlstm_step_kernel(const MlstmArgs a, int cols, int nx, int ny) {
    extern __shared__ __align__(16) float smem[];
    const int dim = (int)a.dim, vdim = (int)a.vdim, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float *qs = smem;                 // [T][dim]
    float *ks = qs + T * dim;         // [T][dim]
    float *nq = ks + T * dim;         // [T][dim] products of n and q
    float *ns = nq + T * dim;         // [dim]
    float *red = ns + dim;            // [T][ny][cols]
    __shared__ float al[T], be[T], em[T];
    __shared__ float ssq[2][T];       // read by the other CTAs of the cluster
    cg::cluster_group cluster = cg::this_cluster();
    const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * cols;
    const int tx = tid % nx, ty = tid / nx, col = c0 + tx * VEC;
    const bool active = ty < ny && col < vdim;
    const size_t bh = (size_t)b * a.H + h;
    float *st = a.state + bh * dim * vdim + col;
    // What the cache holds does not depend on this step's projections: it is requested while they still run.  (No other kernel of a
    // step writes it, and the length changes at the step's end.)
    Cols<VEC> pre[T == 1 ? kPre : 1];
    if (T == 1) {
#pragma unroll
        for (int i = 0; i < kPre; ++i)
            if (active && ty + i * ny < dim) pre[i] = load_cols<VEC>(st + (size_t)(ty + i * ny) * vdim);
    }
    const bool fresh = *a.d_len == 0;
    for (int i = tid; i < dim; i += kThreads) ns[i] = fresh ? 0.f : a.norm[bh * dim + i];
    float m = fresh ? 0.f : a.mx[bh];  // (kept by the first warp)
    pdl_launch();
    pdl_wait();
    const float qscale = rsqrtf_exact((float)dim);
    int buf = 0;
#pragma unroll 1
    for (int t0 = 0; t0 < (int)a.S; t0 += T, buf ^= 1) {
        const int nt = min(T, (int)a.S - t0);
        const size_t row0 = (size_t)b * a.S + t0;
        for (int i = tid; i < nt * dim; i += kThreads) {
            const int t = i / dim, r = i - t * dim;
            const float *u = a.u + (row0 + t) * a.u_ld + (size_t)h * dim + r;
            qs[i] = __fmul_rn(u[0], qscale);
            ks[i] = u[a.u_k];
        }
        if (warp == 0) {
            float li = 0.f, lf = 0.f;
            if (lane < nt) log_gates(a.z + (row0 + lane) * a.z_ld, a.z_bias, (int)a.H, h, a.cap, li, lf);
            float mine = 0.f, before = 0.f;
#pragma unroll
            for (int t = 0; t < T; ++t) {
                const float i_t = __shfl_sync(0xffffffffu, li, t), f_t = __shfl_sync(0xffffffffu, lf, t);
                if (t >= nt) break;
                const float mn = fmaxf(f_t + m, i_t);
                if (lane == t) {
                    before = m;
                    mine = mn;
                }
                m = mn;
            }
            if (lane < nt) {
                al[lane] = expf(lf + before - mine);
                be[lane] = expf(li - mine);
                em[lane] = expf(-mine);
            }
        }
        Cols<VEC> vb[T];
        if (active)
#pragma unroll
            for (int t = 0; t < T; ++t)
#pragma unroll
                for (int k = 0; k < VEC; ++k) vb[t].v[k] = t < nt ? a.u[(row0 + t) * a.u_ld + a.u_v + (size_t)h * vdim + col + k] : 0.f;
        // what the last stage multiplies with (a warp finishes token `warp`; the first two columns of a lane are ready by then)
        float gain[2] = {0.f, 0.f}, gate[2] = {0.f, 0.f};
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int c = lane + 32 * k;
            if (warp < nt && c < cols && c0 + c < vdim) {
                gain[k] = a.head_gain[(size_t)h * vdim + c0 + c];
                gate[k] = a.u[(row0 + warp) * a.u_ld + a.u_g + (size_t)h * vdim + c0 + c];
            }
        }
        __syncthreads();
        for (int r = tid; r < dim; r += kThreads) {
            float n = ns[r];
#pragma unroll
            for (int t = 0; t < T; ++t)
                if (t < nt) {
                    n = fmaf(al[t], n, be[t] * ks[t * dim + r]);
                    nq[t * dim + r] = n * qs[t * dim + r];
                }
            ns[r] = n;
        }
        if (active) {
            Cols<VEC> acc[T];
#pragma unroll
            for (int t = 0; t < T; ++t) {
#pragma unroll
                for (int k = 0; k < VEC; ++k) {
                    if (t < nt) vb[t].v[k] *= be[t];
                    acc[t].v[k] = 0.f;
                }
            }
            auto apply = [&](int r, Cols<VEC> s) {
                if (fresh && t0 == 0)
#pragma unroll
                    for (int k = 0; k < VEC; ++k) s.v[k] = 0.f;
#pragma unroll
                for (int t = 0; t < T; ++t)
                    if (t < nt) {
                        const float d = al[t], kr = ks[t * dim + r], qr = qs[t * dim + r];
#pragma unroll
                        for (int k = 0; k < VEC; ++k) {
                            s.v[k] = fmaf(d, s.v[k], kr * vb[t].v[k]);
                            acc[t].v[k] = fmaf(s.v[k], qr, acc[t].v[k]);
                        }
                    }
                store_cols<VEC>(st + (size_t)r * vdim, s);
            };
            if (T == 1) {
#pragma unroll
                for (int i = 0; i < kPre; ++i)
                    if (ty + i * ny < dim) apply(ty + i * ny, pre[i]);
#pragma unroll 1
                for (int r = ty + kPre * ny; r < dim; r += ny) apply(r, load_cols<VEC>(st + (size_t)r * vdim));
            } else {
#pragma unroll 1
                for (int r = ty; r < dim; r += 4 * ny) {
                    Cols<VEC> s[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (r + i * ny < dim) s[i] = load_cols<VEC>(st + (size_t)(r + i * ny) * vdim);
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (r + i * ny < dim) apply(r + i * ny, s[i]);
                }
            }
#pragma unroll
            for (int t = 0; t < T; ++t)
#pragma unroll
                for (int k = 0; k < VEC; ++k) red[(t * ny + ty) * cols + tx * VEC + k] = acc[t].v[k];
        }
        __syncthreads();
        // warp t finishes token t (T <= 8 warps): denominator, this slice's outputs and their sum of squares
        static_assert(T <= kWarps, "a warp per token");
        const int t = warp;
        float *os = red + (size_t)t * ny * cols;  // (the sums over the row groups replace the first group's)
        if (t < nt) {
            float s = 0.f;
            for (int r = lane; r < dim; r += 32) s += nq[t * dim + r];
            const float den = fmaxf(fabsf(warp_sum(s)), em[t]) + 1e-6f;
            float ss = 0.f;
            for (int c = lane; c < cols; c += 32) {
                float o = 0.f;
                if (c0 + c < vdim) {
#pragma unroll 8
                    for (int y = 0; y < ny; ++y) o += os[y * cols + c];
                    o = __fdiv_rn(o, den);
                }
                os[c] = o;
                ss = fmaf(o, o, ss);
            }
            ss = warp_sum(ss);
            if (lane == 0) ssq[buf][t] = ss;
        }
        cluster.sync();  // (the buffer is rewritten two passes later, after every CTA has been through the next barrier)
        if (t < nt) {
            const float ss = warp_sum(lane < (int)cluster.num_blocks() ? *cluster.map_shared_rank(&ssq[buf][t], lane) : 0.f);
            const float inv = __fdiv_rn(1.0f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)vdim), a.eps)));
            for (int c = lane, k = 0; c < cols && c0 + c < vdim; c += 32, ++k) {
                const size_t j = (size_t)h * vdim + c0 + c, at = (row0 + t) * a.H * vdim + j;
                const float hg = k == 0 ? gain[0] : k == 1 ? gain[1] : a.head_gain[j], g = k == 0 ? gate[0] : k == 1 ? gate[1] : a.u[(row0 + t) * a.u_ld + a.u_g + j];
                const float v = os[c] * inv * hg * sigmoid_f(g);
                if (a.out) a.out[at] = v;
                if (a.out_hi) store_split(v, a.out_hi, a.out_lo, at);
            }
        }
        __syncthreads();
    }
    // every CTA of the cluster has read n and m before its first barrier; none leaves while another still reads its sums
    if (blockIdx.x == 0) {
        for (int i = tid; i < dim; i += kThreads) a.norm[bh * dim + i] = ns[i];
        if (tid == 0) a.mx[bh] = m;
    }
    cluster.sync();
}

template <int VEC, int T>
int launch_step(lumen_ctx *ctx, const MlstmArgs &a, int cols, unsigned slices, cudaStream_t s) {
    const int nx = cols / VEC, ny = kThreads / nx;
    const size_t smem = ((size_t)T * (3 * a.dim + (size_t)ny * cols) + a.dim) * sizeof(float);
    if (smem > 200 * 1024) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "matrix memory: keys of %zu numbers", a.dim);
    if (smem > 48 * 1024) LUMEN_CUDA(ctx, cudaFuncSetAttribute(mlstm_step_kernel<VEC, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return launch_pdl_cluster(ctx, mlstm_step_kernel<VEC, T>, slices, dim3(slices, (unsigned)a.H, (unsigned)a.B), kThreads, smem, s, a, cols, nx, ny);
}

}  // namespace

int launch_mlstm_step(lumen_ctx *ctx, const MlstmArgs &a, cudaStream_t s) {
    // slices of about 32 columns or more, at most 8 of them
    const size_t want = std::max<size_t>(1, std::min<size_t>(8, (a.vdim + 31) / 32));
    const size_t cols = ((a.vdim + want - 1) / want + 3) / 4 * 4;
    const unsigned slices = (unsigned)((a.vdim + cols - 1) / cols);
    if (cols > (size_t)kThreads || a.H > 65535 || a.B > 65535) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "matrix memory: %zu heads with values of %zu numbers", a.H, a.vdim);
    if (a.vdim % 4 == 0) return a.S == 1 ? launch_step<4, 1>(ctx, a, (int)cols, slices, s) : launch_step<4, 8>(ctx, a, (int)cols, slices, s);
    return a.S == 1 ? launch_step<1, 1>(ctx, a, (int)cols, slices, s) : launch_step<1, 8>(ctx, a, (int)cols, slices, s);
}

}  // namespace lumen
