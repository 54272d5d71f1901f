// Routed experts: sigmoid scores, the `top` largest, every chosen expert applied to score * x, plus a shared expert.
//
// Few rows (decode): moe_gate_up_kernel chooses the experts of its row from the router logits (each CTA for itself: a few
// hundred comparisons) and streams the chosen gate and up rows; moe_down_kernel streams the chosen down rows and adds the
// experts' outputs.  The score is applied to the gate and up sums, which are linear in the expert's input.
// Many rows: moe_group_kernel sorts the (row, expert) pairs by expert and lists the 128-row tiles that the grouped
// tensor-core product (gemm_tc.cu) walks.
#include <algorithm>

#include "decoder_kernels.cuh"
#include "gemv_rows.cuh"

namespace lumen {
namespace {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;

// The `top` largest of E scores (ties: the lower index), by one warp.  sc is overwritten.
__device__ __forceinline__ void warp_top(float *sc, int E, int top, int lane, int *sel, float *weight) {
    for (int k = 0; k < top; ++k) {
        float best = -1.f;
        int at = E;
        for (int e = lane; e < E; e += 32)
            if (sc[e] > best) {
                best = sc[e];
                at = e;
            }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (ob > best || (ob == best && oa < at)) {
                best = ob;
                at = oa;
            }
        }
        at = min(at, E - 1);  // (scores that are not numbers choose nothing)
        if (lane == 0) {
            sel[k] = at;
            weight[k] = fmaxf(best, 0.f);
            sc[at] = -1.f;
        }
        __syncwarp();
    }
}

__device__ __forceinline__ size_t gate_row(size_t i) { return i / kGateBlock * (2 * kGateBlock) + i % kGateBlock; }

template <typename WT>
__global__ void __launch_bounds__(kThreads) moe_gate_up_kernel(const MoeArgs a) {
    extern __shared__ __align__(16) float smem[];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int E = (int)a.experts, top = (int)a.top;
    const size_t m = blockIdx.y, K = a.W;
    float *xs = smem, *sc = xs + ((K + 3) & ~(size_t)3), *weight = sc + E;
    int *sel = reinterpret_cast<int *>(weight + top);
    pdl_launch();
    pdl_wait();
    for (size_t k = tid; k < K; k += kThreads) xs[k] = a.x[m * K + k];
    for (int e = tid; e < E; e += kThreads) sc[e] = sigmoid_f(a.z[m * E + e]);
    __syncthreads();
    if (warp == 0) {
        warp_top(sc, E, top, lane, sel, weight);
        if (blockIdx.x == 0)
            for (int k = lane; k < top; k += 32) a.sel[m * top + k] = sel[k];
    }
    __syncthreads();
    const size_t routed = (size_t)top * a.ff, total = routed + a.shared_ff;
    const size_t per_expert = ((a.ff + kGateBlock - 1) / kGateBlock) * 2 * kGateBlock;
    constexpr int VEC = 16 / sizeof(WT);
    const bool vec_ok = K % VEC == 0;  // (matrices of the slab start on 256-byte boundaries)
    for (size_t i = (size_t)blockIdx.x * kWarps + warp; i < total; i += (size_t)gridDim.x * kWarps) {
        const WT *g_row;
        float w = 1.f, limit = a.shared_limit;
        if (i < routed) {
            const size_t slot = i / a.ff, r = i - slot * a.ff;
            g_row = static_cast<const WT *>(a.gate_up) + ((size_t)sel[slot] * per_expert + gate_row(r)) * K;
            w = weight[slot];
            limit = a.limit;
        } else {
            g_row = static_cast<const WT *>(a.shared_gate_up) + gate_row(i - routed) * K;
        }
        const WT *rows[2] = {g_row, g_row + kGateBlock * K};
        float acc[2][1] = {{0.f}, {0.f}};
        if (vec_ok) {
            rows_dot<WT, 1, 2>(rows, xs, K, lane, acc);
        } else {
            acc[0][0] = row_dot_scalar<WT>(rows[0], xs, (int)K, lane);
            acc[1][0] = row_dot_scalar<WT>(rows[1], xs, (int)K, lane);
        }
        const float g = warp_sum(acc[0][0]) * w, u = warp_sum(acc[1][0]) * w;
        if (lane == 0) a.act[m * total + i] = gated_act(g, u, limit);
    }
}

// Four warps share an output row: the chosen experts' rows and the shared one form one sequence of vectors.
constexpr int kDownWarps = 4, kDownRows = kWarps / kDownWarps;
template <typename WT>
__global__ void __launch_bounds__(kThreads, 3) moe_down_kernel(const MoeArgs a) {
    extern __shared__ __align__(16) float act[];  // every expert's activations, each on a 16-byte boundary; then the experts' numbers
    __shared__ float red[kWarps];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = warp % kDownWarps;
    const int top = (int)a.top, ff = (int)a.ff, sff = (int)a.shared_ff, ff4 = (ff + 3) & ~3;
    const size_t m = blockIdx.y, total = (size_t)top * ff + sff;
    int *sel = reinterpret_cast<int *>(act + top * ff4 + ((sff + 3) & ~3));
    constexpr int VEC = 16 / sizeof(WT);
    const bool vec_ok = ff % VEC == 0 && sff % VEC == 0;
    pdl_launch();
    pdl_wait();
    const float *src = a.act + m * total;
    if (ff4 == ff && total % 4 == 0) {
        for (size_t i = tid; i < total / 4; i += kThreads) reinterpret_cast<float4 *>(act)[i] = reinterpret_cast<const float4 *>(src)[i];
    } else {
        for (int k = 0; k <= top; ++k)
            for (int i = tid; i < (k < top ? ff : sff); i += kThreads) act[k * ff4 + i] = src[k * ff + i];
    }
    if (tid < top) sel[tid] = a.sel[m * top + tid];
    for (int k = kThreads + tid; k < top; k += kThreads) sel[k] = a.sel[m * top + k];
    __syncthreads();
    const unsigned nv = (unsigned)(ff / VEC), routed = nv * top, all = routed + (unsigned)(sff / VEC);
    for (size_t base = (size_t)blockIdx.x * kDownRows; base < a.W; base += (size_t)gridDim.x * kDownRows) {
        const size_t n = base + warp / kDownWarps;
        float acc[1] = {0.f};
        if (n < a.W) {
            const WT *shared_row = static_cast<const WT *>(a.shared_down) + n * sff;
            if (vec_ok) {
                for (unsigned i0 = part * 256; i0 < all; i0 += kDownWarps * 256) {
                    uint4 wv[8];
                    int xo[8];
#pragma unroll
                    for (int u = 0; u < 8; ++u) {
                        const unsigned i = i0 + u * 32 + lane;
                        xo[u] = 0;
                        wv[u] = make_uint4(0u, 0u, 0u, 0u);
                        if (i < routed) {
                            const unsigned slot = i / nv, at = i - slot * nv;
                            wv[u] = ld_stream_u4(reinterpret_cast<const uint4 *>(static_cast<const WT *>(a.down) + ((size_t)sel[slot] * a.W + n) * ff) + at);
                            xo[u] = slot * ff4 + at * VEC;
                        } else if (i < all) {
                            wv[u] = ld_stream_u4(reinterpret_cast<const uint4 *>(shared_row) + (i - routed));
                            xo[u] = top * ff4 + (i - routed) * VEC;
                        }
                    }
#pragma unroll
                    for (int u = 0; u < 8; ++u)
                        if (i0 + u * 32 + lane < all) acc[0] = vec_dot<WT>(wv[u], act + xo[u], acc[0]);
                }
            } else {
                for (int k = part; k <= top; k += kDownWarps) {
                    if (k < top) acc[0] += row_dot_scalar<WT>(static_cast<const WT *>(a.down) + ((size_t)sel[k] * a.W + n) * ff, act + k * ff4, ff, lane);
                    else if (sff) acc[0] += row_dot_scalar<WT>(shared_row, act + top * ff4, sff, lane);
                }
            }
        }
        const float v = warp_sum(acc[0]);
        if (lane == 0) red[warp] = v;
        __syncthreads();
        if (lane == 0 && part == 0 && n < a.W) {
            float y = 0.f;
#pragma unroll
            for (int i = 0; i < kDownWarps; ++i) y += red[warp + i];
            a.y[m * a.W + n] = y;
        }
        __syncthreads();
    }
}

// One warp per row.
__global__ void __launch_bounds__(kThreads) moe_choose_kernel(const float *z, int M, int E, int top, int *sel, float *weight) {
    extern __shared__ float sc_all[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int m = blockIdx.x * kWarps + warp;
    if (m >= M) return;
    float *sc = sc_all + (size_t)warp * E;
    for (int e = lane; e < E; e += 32) sc[e] = sigmoid_f(z[(size_t)m * E + e]);
    __syncwarp();
    warp_top(sc, E, top, lane, sel + (size_t)m * top, weight + (size_t)m * top);
}

// One CTA: rows counted per expert, tiles listed, every (row, slot) given its place.
__global__ void __launch_bounds__(1024) moe_group_kernel(const MoeGroupArgs a) {
    extern __shared__ int counts[];  // [E] counts, then [E] cursors
    const int E = (int)a.experts, n = (int)(a.M * a.top), tid = threadIdx.x;
    int *cursor = counts + E;
    for (int e = tid; e < E; e += 1024) counts[e] = 0;
    __syncthreads();
    for (int i = tid; i < n; i += 1024) atomicAdd(&counts[a.sel[i]], 1);
    __syncthreads();
    if (tid == 0) {
        int off = 0, t = 0;
        for (int e = 0; e < E; ++e) {
            cursor[e] = off;
            const int end = off + counts[e];
            for (int r = off; r < end; r += 128) a.tiles[t++] = make_int4(r, end, e, 0);
            off = end;
        }
        *a.n_tiles = t;
    }
    __syncthreads();
    for (int i = tid; i < n; i += 1024) {
        const int p = atomicAdd(&cursor[a.sel[i]], 1);
        a.pos[i] = p;
        a.src[p] = i / (int)a.top;
        a.row_scale[p] = a.weight[i];
    }
}

__global__ void __launch_bounds__(128) gather_rows_kernel(const __nv_bfloat16 *__restrict__ in, const int *__restrict__ src,
                                                          __nv_bfloat16 *__restrict__ out, size_t dim) {
    const size_t r = blockIdx.x;
    const uint4 *from = reinterpret_cast<const uint4 *>(in + (size_t)src[r] * dim);
    uint4 *to = reinterpret_cast<uint4 *>(out + r * dim);
    for (size_t i = threadIdx.x; i < dim / 8; i += 128) to[i] = from[i];
}

size_t gate_up_smem(const MoeArgs &a) { return (((a.W + 3) & ~(size_t)3) + a.experts + 2 * a.top) * sizeof(float); }
size_t down_smem(const MoeArgs &a) { return (a.top * (((a.ff + 3) & ~(size_t)3) + 1) + a.shared_ff + 4) * sizeof(float); }

template <typename WT>
int launch_vec_t(lumen_ctx *ctx, const MoeArgs &a, cudaStream_t s) {
    const size_t s1 = gate_up_smem(a), s2 = down_smem(a);
    if (s1 > 48 * 1024) LUMEN_CUDA(ctx, cudaFuncSetAttribute(moe_gate_up_kernel<WT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1));
    if (s2 > 48 * 1024) LUMEN_CUDA(ctx, cudaFuncSetAttribute(moe_down_kernel<WT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2));
    auto blocks = [&](size_t rows, size_t smem, size_t per_cta) {
        const size_t per_sm = std::max<size_t>(1, std::min<size_t>(8, 227 * 1024 / (smem + 1024)));
        return (unsigned)std::max<size_t>(1, std::min((rows + per_cta - 1) / per_cta, (size_t)ctx->num_sms * per_sm));
    };
    LUMEN_TRY(launch_pdl(ctx, moe_gate_up_kernel<WT>, dim3(blocks(a.top * a.ff + a.shared_ff, s1, kWarps), (unsigned)a.M), kThreads, s1, s, a));
    return launch_pdl(ctx, moe_down_kernel<WT>, dim3(blocks(a.W, s2, kDownRows), (unsigned)a.M), kThreads, s2, s, a);
}

}  // namespace

bool moe_vec_usable(const MoeArgs &a) { return gate_up_smem(a) <= 200 * 1024 && down_smem(a) <= 200 * 1024; }

int launch_moe_vec(lumen_ctx *ctx, const MoeArgs &a, cudaStream_t s) {
    if (!moe_vec_usable(a)) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "experts: width %zu, %zu x %zu", a.W, a.top, a.ff);
    // blockIdx.y carries the row: at most 65535 per launch
    for (size_t m0 = 0; m0 < a.M; m0 += 65535) {
        MoeArgs p = a;
        const size_t total = a.top * a.ff + a.shared_ff;
        p.M = std::min<size_t>(65535, a.M - m0);
        p.x += m0 * a.W; p.z += m0 * a.experts; p.act += m0 * total; p.sel += m0 * a.top; p.y += m0 * a.W;
        LUMEN_TRY(a.wdt == LUMEN_F32 ? launch_vec_t<float>(ctx, p, s) : launch_vec_t<__nv_bfloat16>(ctx, p, s));
    }
    return LUMEN_OK;
}

int launch_moe_group(lumen_ctx *ctx, const MoeGroupArgs &a, cudaStream_t s) {
    const size_t smem = kWarps * a.experts * sizeof(float), gsmem = 2 * a.experts * sizeof(int);
    if (smem > 48 * 1024 || gsmem > 48 * 1024) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "router: %zu experts", a.experts);
    moe_choose_kernel<<<(unsigned)((a.M + kWarps - 1) / kWarps), kThreads, smem, s>>>(a.z, (int)a.M, (int)a.experts, (int)a.top, a.sel, a.weight);
    LUMEN_LAUNCHED(ctx);
    moe_group_kernel<<<1, 1024, gsmem, s>>>(a);
    LUMEN_LAUNCHED(ctx);
    return LUMEN_OK;
}

int launch_gather_rows(lumen_ctx *ctx, const __nv_bfloat16 *in, const int *src, __nv_bfloat16 *out, size_t rows, size_t dim, cudaStream_t s) {
    if (rows == 0) return LUMEN_OK;
    if (dim % 8) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "gather: row length %zu", dim);
    gather_rows_kernel<<<(unsigned)rows, 128, 0, s>>>(in, src, out, dim);
    LUMEN_LAUNCHED(ctx);
    return LUMEN_OK;
}

}  // namespace lumen
