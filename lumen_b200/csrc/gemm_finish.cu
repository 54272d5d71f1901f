// Kernels that finish a tensor-core product of a batched step or a prefill slice in one pass over its split-K slices,
// producing what the NEXT product reads, so that a block of LlamaBlock::forward (src/models/llama.rs:107-115, :59-65)
// needs 11 launches instead of 20:
//   sum_norm_split_kernel  x = sum of slices + residual;  (hi, lo) = bf16 split of RMSNorm(x) * gains
//                          (replaces split-K sum + RMSNorm + hi/lo split)
//   sum_swiglu_split_kernel  (hi, lo) = bf16 split of silu(gate) * up, gate and up being the column halves of one product
//                          over the concatenated gate and up weights (replaces two split-K sums + SiLU*mul + hi/lo split)
#include <algorithm>

#include "decoder_kernels.cuh"
#include "row_finish.cuh"

namespace lumen {
namespace {

__global__ void __launch_bounds__(256) sum_norm_split_kernel(const float *__restrict__ part, int splits, const float *residual, int rows,
                                                             int dim, RowFinish f) {
    __shared__ float red[8];
    const int tid = threadIdx.x, nvec = dim >> 2;
    const size_t mn = (size_t)rows * dim;
    for (int row = blockIdx.x; row < rows; row += gridDim.x) {
        const size_t base = (size_t)row * dim;
        float4 v[kRowVecs];
        row_load_sum(v, part, splits, mn, residual, base, nvec, tid);
        row_finish(v, f, base, dim, nvec, tid, red);
    }
}

// SiLU::forward — src/layers/activation.rs:143-146
__device__ __forceinline__ float silu_mul1(float g, float u) {
    const float sig = __fdiv_rn(1.0f, __fadd_rn(1.0f, expf(-g)));
    return __fmul_rn(__fmul_rn(g, sig), u);
}

// part: [splits][rows][2 * inter]; thread = 4 adjacent columns of one row
__global__ void __launch_bounds__(256) sum_swiglu_split_kernel(const float *__restrict__ part, int splits, size_t rows, size_t inter,
                                                               __nv_bfloat16 *__restrict__ hi, __nv_bfloat16 *__restrict__ lo) {
    const size_t q = (size_t)blockIdx.x * 256 + threadIdx.x, per_row = inter >> 2;
    if (q >= rows * per_row) return;
    const size_t row = q / per_row, col = (q - row * per_row) << 2;
    const size_t mn = rows * 2 * inter, at = row * 2 * inter + col;
    float4 g = *reinterpret_cast<const float4 *>(part + at), u = *reinterpret_cast<const float4 *>(part + at + inter);
#pragma unroll 4
    for (int sl = 1; sl < splits; ++sl) {
        const float4 g2 = *reinterpret_cast<const float4 *>(part + (size_t)sl * mn + at);
        const float4 u2 = *reinterpret_cast<const float4 *>(part + (size_t)sl * mn + at + inter);
        g = add4(g, g2);
        u = add4(u, u2);
    }
    const float4 a = make_float4(silu_mul1(g.x, u.x), silu_mul1(g.y, u.y), silu_mul1(g.z, u.z), silu_mul1(g.w, u.w));
    uint2 h, l;
    split4(a, &h, &l);
    *reinterpret_cast<uint2 *>(hi + row * inter + col) = h;
    *reinterpret_cast<uint2 *>(lo + row * inter + col) = l;
}

// One CTA per row, any row length (the row is kept in shared memory between the passes).  NEXT: the next sublayer reads a norm of
// the new residual.
template <bool NEXT>
__global__ void __launch_bounds__(256) norm_add_kernel(const float *__restrict__ part, int splits, size_t rows, size_t n, const StepFinish f) {
    extern __shared__ __align__(16) float row_s[];
    __shared__ float red[8];
    const int tid = threadIdx.x;
    const size_t row = blockIdx.x, base = row * n, mn = rows * n;
    float ss = 0.f;
    const bool vec = n % 4 == 0;
    if (vec) {
        for (size_t i = tid; i < n / 4; i += 256) {
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
            for (int sl = 0; sl < splits; ++sl) v = add4(v, reinterpret_cast<const float4 *>(part + (size_t)sl * mn + base)[i]);
#pragma unroll 4
            for (int k = 0; k < f.gather_n; ++k) {
                const uint2 g = reinterpret_cast<const uint2 *>(f.gather_src + (size_t)f.gather_idx[row * f.gather_n + k] * n)[i];
                v = add4(v, make_float4(__uint_as_float(g.x << 16), __uint_as_float(g.x & 0xffff0000u), __uint_as_float(g.y << 16),
                                        __uint_as_float(g.y & 0xffff0000u)));
            }
            reinterpret_cast<float4 *>(row_s)[i] = v;
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
    } else {
        for (size_t i = tid; i < n; i += 256) {
            float v = 0.f;
            for (int sl = 0; sl < splits; ++sl) v = __fadd_rn(v, part[(size_t)sl * mn + base + i]);
            for (int k = 0; k < f.gather_n; ++k) v = __fadd_rn(v, __bfloat162float(f.gather_src[(size_t)f.gather_idx[row * f.gather_n + k] * n + i]));
            row_s[i] = v;
            ss = fmaf(v, v, ss);
        }
    }
    auto row_inv = [&](float s) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if ((tid & 31) == 0) red[tid >> 5] = s;
        __syncthreads();
        float t = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) t += red[w];
        __syncthreads();
        return __fdiv_rn(1.0f, sqrtf(__fadd_rn(__fdiv_rn(t, (float)n), f.eps)));
    };
    const float inv = row_inv(ss);
    auto put4 = [&](float4 v, size_t i) {
        if (f.out) reinterpret_cast<float4 *>(f.out + base)[i] = v;
        if (f.hi) {
            uint2 h, l;
            split4(v, &h, &l);
            reinterpret_cast<uint2 *>(f.hi + base)[i] = h;
            if (f.lo) reinterpret_cast<uint2 *>(f.lo + base)[i] = l;
        }
    };
    float ss2 = 0.f;
    if (vec) {
        for (size_t i = tid; i < n / 4; i += 256) {
            const float4 v = reinterpret_cast<const float4 *>(row_s)[i], g = reinterpret_cast<const float4 *>(f.gain)[i];
            float4 *xp = reinterpret_cast<float4 *>(f.x + base) + i;
            const float4 x = add4(*xp, make_float4(__fmul_rn(__fmul_rn(v.x, inv), g.x), __fmul_rn(__fmul_rn(v.y, inv), g.y),
                                                   __fmul_rn(__fmul_rn(v.z, inv), g.z), __fmul_rn(__fmul_rn(v.w, inv), g.w)));
            *xp = x;
            if (NEXT) {
                reinterpret_cast<float4 *>(row_s)[i] = x;
                ss2 = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, ss2))));
            } else {
                put4(x, i);
            }
        }
        if (NEXT) {
            const float inv2 = row_inv(ss2);
            for (size_t i = tid; i < n / 4; i += 256) {
                const float4 x = reinterpret_cast<const float4 *>(row_s)[i], g = reinterpret_cast<const float4 *>(f.next_gain)[i];
                put4(make_float4(__fmul_rn(__fmul_rn(x.x, inv2), g.x), __fmul_rn(__fmul_rn(x.y, inv2), g.y), __fmul_rn(__fmul_rn(x.z, inv2), g.z),
                                 __fmul_rn(__fmul_rn(x.w, inv2), g.w)), i);
            }
        }
        return;
    }
    auto put = [&](float v, size_t i) {
        if (f.out) f.out[base + i] = v;
        if (f.hi) store_split(v, f.hi, f.lo, base + i);
    };
    for (size_t i = tid; i < n; i += 256) {
        const float x = __fadd_rn(f.x[base + i], __fmul_rn(__fmul_rn(row_s[i], inv), f.gain[i]));
        f.x[base + i] = x;
        if (NEXT) {
            row_s[i] = x;
            ss2 = fmaf(x, x, ss2);
        } else {
            put(x, i);
        }
    }
    if (NEXT) {
        const float inv2 = row_inv(ss2);
        for (size_t i = tid; i < n; i += 256) put(__fmul_rn(__fmul_rn(row_s[i], inv2), f.next_gain[i]), i);
    }
}

// One thread per output element.
__global__ void __launch_bounds__(256) act_finish_kernel(const float *__restrict__ part, int splits, size_t rows, size_t n, const StepFinish f) {
    const size_t out_n = f.kind == StepFinish::kGated ? f.ff : n;
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= rows * out_n) return;
    const size_t row = i / out_n, col = i - row * out_n, mn = rows * n;
    auto sum = [&](size_t c) {
        float v = part[row * n + c];
        for (int sl = 1; sl < splits; ++sl) v = __fadd_rn(v, part[(size_t)sl * mn + row * n + c]);
        return v;
    };
    float v;
    if (f.kind == StepFinish::kGated) {
        const size_t at = col / kGateBlock * (2 * kGateBlock) + col % kGateBlock;
        const float g = sum(at), u = sum(at + kGateBlock);
        v = f.glu == StepFinish::kGeluTanh ? gelu_tanh(g) * u : gated_act(g, u, f.limit);
    } else {
        v = sum(col);
        if (f.kind != StepFinish::kStore) v = gelu_tanh(v);
        if (f.kind == StepFinish::kSideGate) {
            const unsigned long long tok = id_to_index(f.ids[row]);
            v *= tok < f.table_rows ? table_at(f.table, f.table_dt, tok * f.table_ld + col) : 0.f;
        }
    }
    if (f.out) f.out[i] = v;
    if (f.hi) store_split(v, f.hi, f.lo, i);
}

}  // namespace

int launch_step_finish(lumen_ctx *ctx, const float *part, int splits, size_t rows, size_t n, const StepFinish &f, cudaStream_t s) {
    if (rows == 0 || n == 0) return LUMEN_OK;
    if (f.kind == StepFinish::kNormAdd) {
        const size_t smem = n * sizeof(float);
        if (smem > 200 * 1024) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "row finisher: row length %zu", n);
        const auto kernel = f.next_gain ? norm_add_kernel<true> : norm_add_kernel<false>;
        if (smem > 48 * 1024) LUMEN_CUDA(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        kernel<<<(unsigned)rows, 256, smem, s>>>(part, part ? splits : 0, rows, n, f);
    } else {
        const size_t total = rows * (f.kind == StepFinish::kGated ? f.ff : n);
        act_finish_kernel<<<(unsigned)((total + 255) / 256), 256, 0, s>>>(part, splits, rows, n, f);
    }
    LUMEN_LAUNCHED(ctx);
    return LUMEN_OK;
}

bool row_finish_usable(size_t dim) { return dim % 8 == 0 && dim <= (size_t)kRowVecs * 1024; }

int launch_sum_norm_split(lumen_ctx *ctx, const float *part, int splits, const float *residual, size_t rows, size_t dim, float *out,
                          const float *norm_w, float eps, __nv_bfloat16 *hi, __nv_bfloat16 *lo, cudaStream_t s) {
    if (rows == 0) return LUMEN_OK;
    if (!row_finish_usable(dim)) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "row finisher: row length %zu", dim);
    RowFinish f{out, norm_w, eps, nullptr, hi, lo};
    const unsigned grid = (unsigned)std::min<size_t>(rows, (size_t)ctx->num_sms * 8);
    sum_norm_split_kernel<<<grid, 256, 0, s>>>(part, splits, residual, (int)rows, (int)dim, f);
    LUMEN_LAUNCHED(ctx);
    return LUMEN_OK;
}

int launch_sum_swiglu_split(lumen_ctx *ctx, const float *part, int splits, size_t rows, size_t inter, __nv_bfloat16 *hi,
                            __nv_bfloat16 *lo, cudaStream_t s) {
    if (rows == 0 || inter == 0) return LUMEN_OK;
    if (inter % 8) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "SwiGLU finisher: intermediate size %zu", inter);
    const size_t quads = rows * (inter >> 2);
    sum_swiglu_split_kernel<<<(unsigned)((quads + 255) / 256), 256, 0, s>>>(part, splits, rows, inter, hi, lo);
    LUMEN_LAUNCHED(ctx);
    return LUMEN_OK;
}

}  // namespace lumen
