// Token inputs of the models given as a list of layers: embedding (scaled, plus a hashed bigram embedding) with the norm that the
// first layer reads, and the end of a step.
#include "decoder_kernels.cuh"
#include "row_finish.cuh"

namespace lumen {
namespace {

template <typename T>
__global__ void __launch_bounds__(256) embed_kernel(EmbedArgs a, DeviceStatus *status) {
    const size_t m = blockIdx.x, b = m / a.S, s = m - b * a.S;
    pdl_launch();
    pdl_wait();
    unsigned long long tok = id_to_index(a.ids[m]);
    if (tok >= a.vocab) {
        if (threadIdx.x == 0 && atomicCAS(&status->code, 0, LUMEN_ERR_EMBED_RANGE) == 0) {
            status->detail0 = (int)m;
            status->detail1 = (int)min(tok, 0x7fffffffull);
        }
        tok = 0;
    }
    const T *row = static_cast<const T *>(a.embed) + tok * a.dim;
    const T *brow = nullptr;
    if (a.bigram) {
        unsigned long long r = a.buckets;
        if (s > 0) r = (id_to_index(a.ids[m - 1]) * a.mul_prev + tok * a.mul_cur) % a.buckets;
        else if (*a.d_len > 0) r = ((unsigned long long)a.last_tok[b] * a.mul_prev + tok * a.mul_cur) % a.buckets;
        brow = static_cast<const T *>(a.bigram) + r * a.dim;
    }
    __shared__ float red[8];
    auto inv_rms = [&](float ss) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) ss += red[w];
        return __fdiv_rn(1.0f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)a.dim), a.eps)));
    };
    float ss = 0.f;
    if (a.dim % 4 == 0 && a.dim <= (size_t)kRowVecs * 1024) {  // the row stays in registers, four numbers at a time
        const int n4 = (int)(a.dim / 4);
        auto load4 = [](const T *p) {
            if constexpr (sizeof(T) == 4) return *reinterpret_cast<const float4 *>(p);
            else {
                const uint2 u = *reinterpret_cast<const uint2 *>(p);
                return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
            }
        };
        float4 v[kRowVecs];
#pragma unroll
        for (int k = 0; k < kRowVecs; ++k) {
            const int i = threadIdx.x + 256 * k;
            if (i >= n4) break;
            const float4 e = load4(row + 4 * i);
            v[k] = make_float4(__fmul_rn(e.x, a.scale), __fmul_rn(e.y, a.scale), __fmul_rn(e.z, a.scale), __fmul_rn(e.w, a.scale));
            if (brow) v[k] = add4(v[k], load4(brow + 4 * i));
            reinterpret_cast<float4 *>(a.x + m * a.dim)[i] = v[k];
            ss = fmaf(v[k].x, v[k].x, fmaf(v[k].y, v[k].y, fmaf(v[k].z, v[k].z, fmaf(v[k].w, v[k].w, ss))));
        }
        const float inv = a.norm_w ? inv_rms(ss) : 1.f;
#pragma unroll
        for (int k = 0; k < kRowVecs; ++k) {
            const int i = threadIdx.x + 256 * k;
            if (i >= n4) break;
            if (a.norm_w) {
                const float4 g = reinterpret_cast<const float4 *>(a.norm_w)[i];
                v[k] = make_float4(__fmul_rn(__fmul_rn(v[k].x, inv), g.x), __fmul_rn(__fmul_rn(v[k].y, inv), g.y), __fmul_rn(__fmul_rn(v[k].z, inv), g.z),
                                   __fmul_rn(__fmul_rn(v[k].w, inv), g.w));
            }
            if (a.out) reinterpret_cast<float4 *>(a.out + m * a.dim)[i] = v[k];
            if (a.hi) {
                uint2 h, l;
                split4(v[k], &h, &l);
                reinterpret_cast<uint2 *>(a.hi + m * a.dim)[i] = h;
                if (a.lo) reinterpret_cast<uint2 *>(a.lo + m * a.dim)[i] = l;
            }
        }
        return;
    }
    auto put = [&](float v, size_t at) {
        if (a.out) a.out[at] = v;
        if (a.hi) store_split(v, a.hi, a.lo, at);
    };
    for (size_t i = threadIdx.x; i < a.dim; i += 256) {
        float v = __fmul_rn(to_f32(row[i]), a.scale);
        if (brow) v = __fadd_rn(v, to_f32(brow[i]));
        const size_t at = m * a.dim + i;
        a.x[at] = v;
        if (a.norm_w) ss = fmaf(v, v, ss);
        else put(v, at);
    }
    if (!a.norm_w) return;
    const float inv = inv_rms(ss);
    for (size_t i = threadIdx.x; i < a.dim; i += 256) {  // (every thread reads back what it wrote)
        const size_t at = m * a.dim + i;
        put(__fmul_rn(__fmul_rn(a.x[at], inv), a.norm_w[i]), at);
    }
}

__global__ void advance_kernel(int *lens, int layers, const float *ids, int *last_tok, int B, int S) {
    pdl_wait();
    for (int l = threadIdx.x; l < layers; l += blockDim.x) lens[l] += S;
    for (int b = threadIdx.x; b < B; b += blockDim.x) last_tok[b] = (int)id_to_index(ids[(size_t)b * S + S - 1]);
}

}  // namespace

int launch_embed(lumen_ctx *ctx, const EmbedArgs &a, cudaStream_t s) {
    const unsigned rows = (unsigned)(a.B * a.S);
    return launch_pdl(ctx, a.dt == LUMEN_F32 ? embed_kernel<float> : embed_kernel<__nv_bfloat16>, rows, 256, 0, s, a, ctx->d_status);
}

int launch_advance(lumen_ctx *ctx, int *d_lens, size_t layers, const float *ids, int *last_tok, size_t B, size_t S, cudaStream_t s) {
    return launch_pdl(ctx, advance_kernel, 1, 256, 0, s, d_lens, (int)layers, ids, last_tok, (int)B, (int)S);
}

}  // namespace lumen
