// Grouped-query attention over chunks: per-head RMS norm and partial rotation of queries and keys, a cache of keys and values
// of sizes of their own (f32, or bf16 in bf16 models), a sink per head in the denominator, a sigmoid gate per head.  A position
// sees the keys of its own chunk up to itself; chunks are counted from position 0, so a piece of the context is found from
// the position alone, however the sequence was cut into steps.
//
//   grouped_append_kernel   keys and values of the step -> cache (and queries as the tensor-core kernel reads them)
//   grouped_rows_kernel     scores, running softmax and weighted values of one row's pieces in 32-bit FMAs, any sizes; f32 models, and
//                           sizes that the MMA kernel (grouped_attn_mma.cu) does not take; in decode steps it appends the new row
//   grouped_merge_kernel    pieces and sink merged, gate applied
// Whole portions run on the tensor cores (attn_prefill_tc.cu).
#include <algorithm>

#include "attn_decode.cuh"
#include "grouped_attention.cuh"

namespace lumen {
namespace {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;

// The same in registers, four neighbouring elements per lane (dim <= 128, everything a multiple of four): every load is issued
// at once, the other half of a pair comes from another lane.
__device__ __forceinline__ float4 head_norm_rotate4(const float *src, int dim, const float *gain, float eps, int rot_dims, const float *cos_row,
                                                    const float *sin_row, int lane) {
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const int e = 4 * lane, half = rot_dims / 2;
    const bool in = e < dim, turns = e < rot_dims;
    const float4 v = in ? *reinterpret_cast<const float4 *>(src + e) : zero, g = in ? *reinterpret_cast<const float4 *>(gain + e) : zero;
    const int p = e < half ? e : e - half;
    const float4 c = turns ? *reinterpret_cast<const float4 *>(cos_row + p) : zero, s = turns ? *reinterpret_cast<const float4 *>(sin_row + p) : zero;
    const float ss = attn_warp_sum(fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))));
    const float inv = __fdiv_rn(1.0f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)dim), eps)));
    float x[4] = {__fmul_rn(__fmul_rn(v.x, inv), g.x), __fmul_rn(__fmul_rn(v.y, inv), g.y), __fmul_rn(__fmul_rn(v.z, inv), g.z),
                  __fmul_rn(__fmul_rn(v.w, inv), g.w)};
    const float cv[4] = {c.x, c.y, c.z, c.w}, sv[4] = {s.x, s.y, s.z, s.w};
    const int other = (e < half ? e + half : e - half) / 4 & 31;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const float y = __shfl_sync(0xffffffffu, x[k], other);
        if (turns) x[k] = e < half ? __fsub_rn(__fmul_rn(x[k], cv[k]), __fmul_rn(y, sv[k])) : __fadd_rn(__fmul_rn(x[k], cv[k]), __fmul_rn(y, sv[k]));
    }
    return make_float4(x[0], x[1], x[2], x[3]);
}
template <typename T>
__device__ __forceinline__ void store4(T *p, float4 v) {
    if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4 *>(p) = v;
    } else {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
    }
}

// Portions: one warp per (row, key head), and with q per (padded row, query head): q[B, H, s_pad, width] bf16, zeros elsewhere.
// VEC: head_norm_rotate4.
template <typename T, bool VEC>
__global__ void __launch_bounds__(kThreads) grouped_append_kernel(const GroupedArgs a, unsigned kv_items, __nv_bfloat16 *q, unsigned s_pad, int width) {
    extern __shared__ __align__(16) float smem[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, dim = (int)a.dim, vdim = (int)a.vdim;
    float *buf = smem + warp * dim;
    unsigned i = blockIdx.x * kWarps + warp;  // (fewer than 2^32 items, see the launcher)
    const unsigned S = (unsigned)a.S, H = (unsigned)a.H, G = (unsigned)a.G;
    const size_t half = a.rot_dims / 2;
    if (i >= kv_items) {
        i -= kv_items;
        const unsigned bs = i / H, h = i - bs * H, b = bs / s_pad, s = bs - b * s_pad;
        if (!q || b >= a.B) return;
        const size_t pos = a.past + s;
        __nv_bfloat16 *row = q + ((size_t)(b * H + h) * s_pad + s) * width;
        const float *src = a.u + (size_t)(b * S + s) * a.u_ld + h * dim, *cos_row = a.cos_t + pos * half, *sin_row = a.sin_t + pos * half;
        if (VEC) {
            const float4 v = s < S ? head_norm_rotate4(src, dim, a.q_gain, a.eps, (int)a.rot_dims, cos_row, sin_row, lane) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (4 * lane < width) store4(row + 4 * lane, v);  // (lanes beyond dim hold zeros)
            return;
        }
        if (s < S) head_norm_rotate(buf, src, dim, a.q_gain, a.eps, (int)a.rot_dims, cos_row, sin_row, lane);
        for (int e = lane; e < width; e += 32) row[e] = __float2bfloat16_rn(s < S && e < dim ? buf[e] : 0.f);
        return;
    }
    const unsigned m = i / G, g = i - m * G, b = m / S;
    const size_t pos = a.past + (m - b * S);
    const float *u = a.u + m * a.u_ld, *ks = u + a.u_k + g * dim, *vs = u + a.u_v + g * vdim;
    const float *cos_row = a.cos_t + pos * half, *sin_row = a.sin_t + pos * half;
    const size_t row = (size_t)(b * G + g) * a.max_seq + pos;
    T *k = static_cast<T *>(a.k) + row * dim, *v = static_cast<T *>(a.v) + row * vdim;
    if (VEC) {
        const bool mine = 4 * lane < vdim;
        const float4 val = mine ? *reinterpret_cast<const float4 *>(vs + 4 * lane) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 key = head_norm_rotate4(ks, dim, a.k_gain, a.eps, (int)a.rot_dims, cos_row, sin_row, lane);
        if (4 * lane < dim) store4(k + 4 * lane, key);
        if (mine) store4(v + 4 * lane, val);
        return;
    }
    head_norm_rotate(buf, ks, dim, a.k_gain, a.eps, (int)a.rot_dims, cos_row, sin_row, lane);
    for (int e = lane; e < dim; e += 32) k[e] = from_f32<T>(buf[e]);
    for (int e = lane; e < vdim; e += 32) v[e] = from_f32<T>(vs[e]);
}

// Two neighbouring elements of a cached row as they lie there.
template <typename T>
struct Pair {
    using Raw = uint32_t;
    static __device__ __forceinline__ Raw pack(float x, float y) {
        const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
        return *reinterpret_cast<const Raw *>(&v);
    }
    static __device__ __forceinline__ float2 get(Raw r) { return make_float2(__uint_as_float(r << 16), __uint_as_float(r & 0xffff0000u)); }
};
template <>
struct Pair<float> {
    using Raw = float2;
    static __device__ __forceinline__ Raw pack(float x, float y) { return make_float2(x, y); }
    static __device__ __forceinline__ float2 get(Raw r) { return r; }
};

__host__ __device__ constexpr int rows_in_flight(int ni) { return ni <= 1 ? 8 : ni == 2 ? 4 : ni <= 4 ? 2 : 1; }

// grid (pieces, G * (H / G / GT), rows): GT query heads of one key head against one piece of the row's chunk.  A lane holds the
// element pairs lane + 32 i, i < NI, of keys and values.  EVEN: dim and vdim are even (pairs are loaded as one).
template <typename T, int GT, int NI, bool EVEN>
__global__ void __launch_bounds__(kThreads) grouped_rows_kernel(const GroupedArgs a, int append) {
    using P = Pair<T>;
    using Raw = typename P::Raw;
    extern __shared__ __align__(16) float smem[];
    constexpr int UN = rows_in_flight(NI), NV = UN * GT;
    const int dim = (int)a.dim, vdim = (int)a.vdim, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float *qs = smem;                       // [GT][dim]
    float *knew = qs + GT * dim;            // [dim]
    float *wm = knew + dim;                 // [warps][GT]
    float *wl = wm + kWarps * GT;           // [warps][GT]
    float *wsoft = wl + kWarps * GT;        // [warps][NV + GT]
    float *wctx = wsoft + kWarps * (NV + GT);  // [warps][GT][vdim]
    const int R = (int)(a.H / a.G), groups = R / GT, hk = (int)blockIdx.y / groups, h0 = hk * R + ((int)blockIdx.y % groups) * GT;
    pdl_launch();
    // A step's own kernels write no cached row but the appended one, and the length only at its end: a layer that appends requests its
    // first rows while the projections still run.
    bool ahead = append;
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
        const T *kbase = static_cast<const T *>(a.k) + (b * a.G + hk) * a.max_seq * dim;
        const T *vbase = static_cast<const T *>(a.v) + (b * a.G + hk) * a.max_seq * vdim;
        const float *u = a.u + m * a.u_ld;
        Raw kra[UN][NI], vra[UN][NI], krb[UN][NI], vrb[UN][NI];
        auto load_pair = [&](const T *row, int n, int e, bool ok) -> Raw {
            if constexpr (EVEN) return ok && e < n ? __ldcg(reinterpret_cast<const Raw *>(row + e)) : P::pack(0.f, 0.f);
            else return P::pack(ok && e < n ? to_f32(row[e]) : 0.f, ok && e + 1 < n ? to_f32(row[e + 1]) : 0.f);
        };
        auto load_rows = [&](int jb, Raw (&kr)[UN][NI], Raw (&vr)[UN][NI]) {
#pragma unroll
            for (int r = 0; r < UN; ++r) {
                const int j = jb + r;
                const bool ok = j < j1 && !(append && j == pos);  // (an appended row comes from the projections)
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const int e = 2 * (lane + 32 * i);
                    kr[r][i] = load_pair(kbase + (size_t)j * dim, dim, e, ok);
                    vr[r][i] = load_pair(vbase + (size_t)j * vdim, vdim, e, ok);
                }
            }
        };
        int jb = j0 + warp * UN;
        if (jb < j1) load_rows(jb, kra, vra);
        if (ahead) pdl_wait();
        ahead = false;
        const size_t half = a.rot_dims / 2;
        const float *cos_row = a.cos_t + pos * half, *sin_row = a.sin_t + pos * half;
        for (int g = warp; g < GT; g += kWarps)
            head_norm_rotate(qs + g * dim, u + (size_t)(h0 + g) * dim, dim, a.q_gain, a.eps, (int)a.rot_dims, cos_row, sin_row, lane);
        const float *vnew = u + a.u_v + (size_t)hk * vdim;
        if (append && j1 == pos + 1 && warp == kWarps - 1) {
            head_norm_rotate(knew, u + a.u_k + (size_t)hk * dim, dim, a.k_gain, a.eps, (int)a.rot_dims, cos_row, sin_row, lane);
            if ((int)blockIdx.y % groups == 0) {
                T *k_row = const_cast<T *>(kbase) + (size_t)pos * dim, *v_row = const_cast<T *>(vbase) + (size_t)pos * vdim;
                for (int e = lane; e < dim; e += 32) k_row[e] = from_f32<T>(knew[e]);
                for (int e = lane; e < vdim; e += 32) v_row[e] = from_f32<T>(vnew[e]);
            }
        }
        __syncthreads();

        // A batch of UN rows x GT heads: the NV dot products are summed across the lanes by one butterfly, after which
        // a lane holds HELD of them; GS lanes hold the scores of one head (see attn_decode.cuh).
        constexpr int HELD = NV >= 32 ? NV / 32 : 1, DUP = NV >= 32 ? 1 : 32 / NV, GS = 32 / GT;
        const int idx0 = NV >= 32 ? lane * HELD : lane / DUP, g_l = idx0 / UN;
        const bool canonical = (lane % DUP) == 0;
        float *ws = wsoft + warp * (NV + GT);
        float2 q[GT][NI], ctx[GT][NI];
        float m_h = -INFINITY, l_h = 0.f;
#pragma unroll
        for (int g = 0; g < GT; ++g)
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int e = 2 * (lane + 32 * i);
                q[g][i] = make_float2(e < dim ? qs[g * dim + e] : 0.f, e + 1 < dim ? qs[g * dim + e + 1] : 0.f);
                ctx[g][i] = make_float2(0.f, 0.f);
            }
        auto do_rows = [&](int jr, Raw (&kr)[UN][NI], Raw (&vr)[UN][NI]) {
            if (append && pos >= jr && pos < jr + UN) {
#pragma unroll
                for (int r = 0; r < UN; ++r)
                    if (jr + r == pos)
#pragma unroll
                        for (int i = 0; i < NI; ++i) {  // (rounded as the cache holds it)
                            const int e = 2 * (lane + 32 * i);
                            kr[r][i] = P::pack(e < dim ? knew[e] : 0.f, e + 1 < dim ? knew[e + 1] : 0.f);
                            vr[r][i] = P::pack(e < vdim ? vnew[e] : 0.f, e + 1 < vdim ? vnew[e + 1] : 0.f);
                        }
            }
            float d[NV];
#pragma unroll
            for (int g = 0; g < GT; ++g)
#pragma unroll
                for (int r = 0; r < UN; ++r) {
                    float s = 0.f;
#pragma unroll
                    for (int i = 0; i < NI; ++i) {
                        const float2 k = P::get(kr[r][i]);
                        s = fmaf(q[g][i].x, k.x, s);
                        s = fmaf(q[g][i].y, k.y, s);
                    }
                    d[g * UN + r] = s;
                }
            attn_reduce_multi<NV>(d, lane);
            float sc[HELD], cmax = -INFINITY;
#pragma unroll
            for (int k = 0; k < HELD; ++k) {
                sc[k] = jr + (idx0 + k) % UN < j1 ? __fmul_rn(d[k], a.scale) : -INFINITY;
                cmax = fmaxf(cmax, sc[k]);
            }
#pragma unroll
            for (int o = 1; o < GS; o <<= 1) cmax = fmaxf(cmax, __shfl_xor_sync(0xffffffffu, cmax, o));
            const float mn = fmaxf(m_h, cmax), r = expf(m_h - mn);  // finite: the batch's first row is inside the piece
            float wsum = 0.f;
#pragma unroll
            for (int k = 0; k < HELD; ++k) {
                const float w = expf(sc[k] - mn);
                if (canonical) ws[idx0 + k] = w;
                wsum += w;
            }
            l_h = fmaf(l_h, r, canonical ? wsum : 0.f);
            m_h = mn;
            if ((lane & (GS - 1)) == 0) ws[NV + g_l] = r;
            __syncwarp();
#pragma unroll
            for (int g = 0; g < GT; ++g) {
                const float rg = ws[NV + g];
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    ctx[g][i].x *= rg;
                    ctx[g][i].y *= rg;
                }
#pragma unroll
                for (int rr = 0; rr < UN; ++rr) {
                    const float w = ws[g * UN + rr];
#pragma unroll
                    for (int i = 0; i < NI; ++i) {
                        const float2 v = P::get(vr[rr][i]);
                        ctx[g][i].x = fmaf(w, v.x, ctx[g][i].x);
                        ctx[g][i].y = fmaf(w, v.y, ctx[g][i].y);
                    }
                }
            }
            __syncwarp();  // the weights are overwritten by the next batch
        };
        constexpr int kStep = kWarps * UN;
        while (jb < j1) {  // the next batch is always in flight
            if (jb + kStep < j1) load_rows(jb + kStep, krb, vrb);
            do_rows(jb, kra, vra);
            jb += kStep;
            if (jb >= j1) break;
            if (jb + kStep < j1) load_rows(jb + kStep, kra, vra);
            do_rows(jb, krb, vrb);
            jb += kStep;
        }
#pragma unroll
        for (int o = 1; o < GS; o <<= 1) l_h += __shfl_xor_sync(0xffffffffu, l_h, o);
        if ((lane & (GS - 1)) == 0) {
            wm[warp * GT + g_l] = m_h;
            wl[warp * GT + g_l] = l_h;
        }
#pragma unroll
        for (int g = 0; g < GT; ++g)
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int e = 2 * (lane + 32 * i);
                if (e < vdim) wctx[(warp * GT + g) * vdim + e] = ctx[g][i].x;
                if (e + 1 < vdim) wctx[(warp * GT + g) * vdim + e + 1] = ctx[g][i].y;
            }
        __syncthreads();
        for (int i = tid; i < GT * vdim; i += kThreads) {
            const int g = i / vdim, e = i - g * vdim;
            float M = -INFINITY, L = 0.f, c = 0.f;
#pragma unroll
            for (int w = 0; w < kWarps; ++w) M = fmaxf(M, wm[w * GT + g]);
#pragma unroll
            for (int w = 0; w < kWarps; ++w) {
                const float mw = wm[w * GT + g], f = mw == -INFINITY ? 0.f : expf(mw - M);
                L = fmaf(wl[w * GT + g], f, L);
                c = fmaf(wctx[(w * GT + g) * vdim + e], f, c);
            }
            const size_t o = (m * a.H + h0 + g) * a.nsplit + blockIdx.x;
            a.part_ctx[o * vdim + e] = c;
            if (e == 0) {
                a.part_ml[o * 2] = M;
                a.part_ml[o * 2 + 1] = L;
            }
        }
        __syncthreads();
    }
}

// grid (heads, rows)
constexpr int kMergeThreads = 128, kMaxPieces = 128;
__global__ void __launch_bounds__(kMergeThreads) grouped_merge_kernel(const GroupedArgs a) {
    __shared__ float w_s[kMaxPieces];
    const size_t h = blockIdx.x;
    const int vdim = (int)a.vdim;
    pdl_launch();
    pdl_wait();
    for (size_t m = blockIdx.y; m < a.B * a.S; m += gridDim.y) {
        const size_t b = m / a.S, row = m * a.H + h;
        const int pos = *a.d_len + (int)(m - b * a.S), len = pos + 1 - chunk_start(pos, a.chunk), per = piece_rows(len, a.nsplit);
        const int pieces = (len + per - 1) / per;
        const float2 *ml = reinterpret_cast<const float2 *>(a.part_ml) + row * a.nsplit;
        const float *ctx = a.part_ctx + row * a.nsplit * vdim;
        const int e0 = threadIdx.x;
        float first[8];  // requested before the weights are known
#pragma unroll
        for (int i = 0; i < 8; ++i) first[i] = i < pieces && e0 < vdim ? ctx[(size_t)i * vdim + e0] : 0.f;
        // every warp finds the maximum and the sum for itself, a piece per lane (grouped_pick_splits: at most kMaxPieces)
        const int lane = threadIdx.x & 31;
        float mx[kMaxPieces / 32], sum[kMaxPieces / 32], M = a.sink[h], L = 0.f;
#pragma unroll
        for (int k = 0; k < kMaxPieces / 32; ++k) {
            const float2 v = lane + 32 * k < pieces ? ml[lane + 32 * k] : make_float2(-INFINITY, 0.f);
            mx[k] = v.x;
            sum[k] = v.y;
            M = fmaxf(M, v.x);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
#pragma unroll
        for (int k = 0; k < kMaxPieces / 32; ++k) {
            mx[k] = expf(mx[k] - M);
            L = fmaf(sum[k], mx[k], L);
        }
        L = attn_warp_sum(L) + expf(a.sink[h] - M);
        if (threadIdx.x < 32)
#pragma unroll
            for (int k = 0; k < kMaxPieces / 32; ++k)
                if (lane + 32 * k < pieces) w_s[lane + 32 * k] = mx[k];
        __syncthreads();
        const float f = __fdiv_rn(sigmoid_f(a.u[m * a.u_ld + a.u_gate + h]), L);
        for (int e = e0; e < vdim; e += kMergeThreads) {
            float c = 0.f;
#pragma unroll
            for (int i = 0; i < 8; ++i)
                if (i < pieces) c = fmaf(e == e0 ? first[i] : ctx[(size_t)i * vdim + e], w_s[i], c);
#pragma unroll 8
            for (int i = 8; i < pieces; ++i) c = fmaf(ctx[(size_t)i * vdim + e], w_s[i], c);
            c *= f;
            if (a.out) a.out[row * vdim + e] = c;
            if (a.out_hi) store_split(c, a.out_hi, a.out_lo, row * vdim + e);
        }
        __syncthreads();  // the weights are overwritten by the next row
    }
}

// grid (row tiles of 64, column tiles of 64, matrices)
__global__ void __launch_bounds__(256) transpose_rows_kernel(const __nv_bfloat16 *__restrict__ in, size_t in_rows, int cols, size_t row0, int rows,
                                                             __nv_bfloat16 *__restrict__ out, size_t pitch) {
    __shared__ __nv_bfloat16 tile[64][66];
    const int r0 = blockIdx.x * 64, c0 = blockIdx.y * 64;
    const size_t mat = blockIdx.z;
    for (int i = threadIdx.x; i < 64 * 64; i += 256) {
        const int r = i >> 6, c = i & 63;
        tile[r][c] = r0 + r < rows && c0 + c < cols ? in[(mat * in_rows + row0 + r0 + r) * cols + c0 + c] : __float2bfloat16_rn(0.f);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < 64 * 64; i += 256) {
        const int c = i >> 6, r = i & 63;
        if (c0 + c < cols && (size_t)(r0 + r) < pitch) out[(mat * cols + c0 + c) * pitch + r0 + r] = tile[r][c];
    }
}

template <typename T, int GT, int NI, bool EVEN>
int launch_rows(lumen_ctx *ctx, const GroupedArgs &a, bool append, cudaStream_t s) {
    constexpr int NV = rows_in_flight(NI) * GT;
    const size_t smem = ((GT + 1) * a.dim + 2 * kWarps * GT + kWarps * (NV + GT) + (size_t)kWarps * GT * a.vdim) * sizeof(float);
    if (smem > 48 * 1024) LUMEN_CUDA(ctx, cudaFuncSetAttribute(grouped_rows_kernel<T, GT, NI, EVEN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const dim3 grid((unsigned)a.nsplit, (unsigned)(a.H / GT), (unsigned)std::min<size_t>(a.B * a.S, 65535));
    return launch_pdl(ctx, grouped_rows_kernel<T, GT, NI, EVEN>, grid, kThreads, smem, s, a, append ? 1 : 0);
}
template <typename T, int GT>
int launch_rows_g(lumen_ctx *ctx, const GroupedArgs &a, bool append, cudaStream_t s) {
    const size_t n = std::max(a.dim, a.vdim);
    if (a.dim % 2 || a.vdim % 2) {
        if (n <= 64) return launch_rows<T, GT, 1, false>(ctx, a, append, s);
        if (n <= 256) return launch_rows<T, GT, 4, false>(ctx, a, append, s);
        return launch_rows<T, 1, 8, false>(ctx, a, append, s);
    }
    if (n <= 64) return launch_rows<T, GT, 1, true>(ctx, a, append, s);
    if (n <= 128) return launch_rows<T, GT, 2, true>(ctx, a, append, s);
    if (n <= 256) return launch_rows<T, GT, 4, true>(ctx, a, append, s);
    return launch_rows<T, 1, 8, true>(ctx, a, append, s);
}
int group_of(const GroupedArgs &a) {  // query heads a CTA takes
    const size_t r = a.H / a.G;
    return std::max(a.dim, a.vdim) > 256 ? 1 : r % 4 == 0 ? 4 : r % 2 == 0 ? 2 : 1;
}

}  // namespace

// As many CTAs as the device holds, pieces that give every warp something, partial results within the workspace (see
// ensure_workspace).
int grouped_pick_splits(const GroupedArgs &a, int num_sms) {
    const bool mma = grouped_mma_usable(a);
    const size_t rows = a.B * a.S, r = a.H / a.G, items = rows * a.G * (mma ? (r + kMmaHeads - 1) / kMmaHeads : r / group_of(a));
    const size_t total = a.past + a.S, len = a.chunk ? std::min(total, a.chunk) : total, piece = mma ? 128 : 64;
    size_t most = std::max<size_t>(1, mma ? num_sms / items : (2 * (size_t)num_sms + items - 1) / items);
    most = std::min(std::min(most, (size_t)kMaxPieces), std::max<size_t>(1, (size_t)num_sms * 64 / (rows * a.H)));
    const size_t n = (len + piece - 1) / piece;
    if (n >= most) return (int)most;
    size_t p = 1;  // few distinct counts while the context grows: every one of them is a graph of its own
    while (p * 2 <= n) p *= 2;
    return (int)p;
}

int launch_grouped_append(lumen_ctx *ctx, const GroupedArgs &a, __nv_bfloat16 *q, size_t s_pad, size_t width, cudaStream_t s) {
    const size_t kv_items = a.own_kv ? a.B * a.S * a.G : 0, items = kv_items + (q ? a.B * s_pad * a.H : 0);
    if (items == 0) return LUMEN_OK;
    if (items >= ((size_t)1 << 31)) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "attention: %zu head vectors in one step", items);
    // (width is a multiple of 64, so it is at most 128 where dim is)
    const bool vec = a.dim <= 128 && a.vdim <= 128 && a.dim % 4 == 0 && a.vdim % 4 == 0 && a.rot_dims % 8 == 0 && a.u_ld % 4 == 0;
    const auto kernel = a.dt == LUMEN_F32 ? (vec ? grouped_append_kernel<float, true> : grouped_append_kernel<float, false>)
                                          : (vec ? grouped_append_kernel<__nv_bfloat16, true> : grouped_append_kernel<__nv_bfloat16, false>);
    kernel<<<(unsigned)((items + kWarps - 1) / kWarps), kThreads, vec ? 0 : kWarps * a.dim * sizeof(float), s>>>(a, (unsigned)kv_items, q, (unsigned)s_pad, (int)width);
    LUMEN_LAUNCHED(ctx);
    return LUMEN_OK;
}

int launch_grouped_attention(lumen_ctx *ctx, const GroupedArgs &a, bool append, cudaStream_t s) {
    if (std::max(a.dim, a.vdim) > kGroupedMaxDim) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "attention: heads of %zu / %zu numbers", a.dim, a.vdim);
    const bool f32 = a.dt == LUMEN_F32;
    int rc;
    if (grouped_mma_usable(a)) rc = launch_grouped_mma(ctx, a, append, s);
    else switch (group_of(a)) {
        case 4: rc = f32 ? launch_rows_g<float, 4>(ctx, a, append, s) : launch_rows_g<__nv_bfloat16, 4>(ctx, a, append, s); break;
        case 2: rc = f32 ? launch_rows_g<float, 2>(ctx, a, append, s) : launch_rows_g<__nv_bfloat16, 2>(ctx, a, append, s); break;
        default: rc = f32 ? launch_rows_g<float, 1>(ctx, a, append, s) : launch_rows_g<__nv_bfloat16, 1>(ctx, a, append, s); break;
    }
    if (rc != LUMEN_OK) return rc;
    return launch_pdl(ctx, grouped_merge_kernel, dim3((unsigned)a.H, (unsigned)std::min<size_t>(a.B * a.S, 65535)), kMergeThreads, 0, s, a);
}

int launch_transpose_rows(lumen_ctx *ctx, const __nv_bfloat16 *in, size_t in_rows, size_t cols, size_t mats, size_t row0, size_t rows,
                          __nv_bfloat16 *out, size_t pitch, cudaStream_t s) {
    transpose_rows_kernel<<<dim3((unsigned)((pitch + 63) / 64), (unsigned)((cols + 63) / 64), (unsigned)mats), 256, 0, s>>>(in, in_rows, (int)cols, row0, (int)rows, out, pitch);
    LUMEN_LAUNCHED(ctx);
    return LUMEN_OK;
}

}  // namespace lumen
