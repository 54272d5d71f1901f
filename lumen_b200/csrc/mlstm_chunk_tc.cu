// Matrix-memory layers over whole portions, in chunks of 128 tokens on the 5th-generation tensor cores (bf16 projections).
//
// Within a chunk that starts with memory S_0, normaliser n_0 and running maximum m_0, let F_t be the sum of the log forget gates up to
// token t, a_t = i_t - F_t and M_t = max(m_0, a_1 .. a_t).  Then m_t = F_t + M_t and, with every exponent at most 0,
//   o_t numerator   = sum_{s <= t} exp(a_s - M_t) (q_t . k_s) v_s + exp(m_0 - M_t) S_0^T q_t
//   n_t . q_t       = sum_{s <= t} exp(a_s - M_t) (q_t . k_s)     + exp(m_0 - M_t) n_0 . q_t
//   S at the end    = exp(m_0 - M_T) S_0 + sum_s exp(a_s - M_T) k_s v_s^T
//   mlstm_scan_kernel    gates, F, M and the weights above, in 32-bit; the maximum is carried from chunk to chunk
//   mlstm_pack_kernel    (exp(a_s - M_T) k_s)^T and v^T, tokens contiguous; the chunk's sum for n
//   mlstm_state_kernel   S^T at the start of every chunk: a CTA owns a tile of S^T [128 values, 64 keys] in 32-bit registers and adds
//                        one product of two transposed operands per chunk, two accumulators of which are in flight
//   mlstm_out_kernel     a CTA owns a chunk of one head: scores, weights (as the attention kernel has its softmax), and per 128
//                        values the products with S_0 and with v
//   mlstm_finish_kernel  norm of every head, gain, output gate
// What 16 bits would lose (weighted keys, S_0, score weights) enters the products as bf16 hi + lo pairs.
//
// Every wait is bounded; a wait that gives up records LUMEN_ERR_TIMEOUT, the CTA runs through without waiting, lets the copies in
// flight land, frees its tensor memory and returns.
#include <algorithm>

#include "decoder_kernels.cuh"
#include "mlstm_gates.cuh"
#include "tc_common.cuh"

namespace lumen {
namespace {

using namespace tc;

constexpr int kC = kMlstmChunk;
constexpr int kSegChunks = 64;  // chunks whose memories are kept at a time
constexpr int kWorkers = 256, kTcThreads = kWorkers + 64;
constexpr float kLog2e = 1.4426950408889634f;

// A segment: T tokens from t0 on of every sequence, in n_chunks chunks; arrays of one number per (b * H + h, token) have a pitch
// of n_chunks * 128.
struct Seg {
    int B, S, H, dim, vdim, t0, T, n_chunks, fresh;
    const __nv_bfloat16 *u;
    size_t u_ld, u_k, u_v, u_g;
    float *a2, *m2, *g, *en, *w;   // a log2(e), M log2(e), exp(m_0 - M), exp(-m), exp(a - M_T)
    float *decay;                  // [B * H, n_chunks] exp(m_0 - M_T)
    __nv_bfloat16 *kt_hi, *kt_lo, *vt;  // [B * H, dim | vdim, pitch]
    float *nsum, *nst;             // [B * H, n_chunks, dim]: the chunk's sum, n_0
    __nv_bfloat16 *s_hi, *s_lo;    // [B * H, n_chunks, vdim, dim] S_0^T
    float *state, *norm;
    __nv_bfloat16 *o;              // [B * T, H * vdim]
    float *ssq;                    // [B * T, H, 2 * tiles]
    int tiles;
    float qscale;
    DeviceStatus *status;
};

// grid B * H, 32 warps: a warp scans a chunk (4 tokens per lane), then the chunks' maxima are chained.
__global__ void __launch_bounds__(1024) mlstm_scan_kernel(const MlstmArgs a, const Seg p) {
    __shared__ float f_end[kSegChunks], a_max[kSegChunks], m_0[kSegChunks];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, bh = blockIdx.x, b = bh / p.H, h = bh - b * p.H;
    constexpr int NC = kSegChunks / 32;
    float F[NC][4], A[NC][4], cm[NC][4];  // sum of log forget gates, a, running maximum of a
#pragma unroll
    for (int i = 0; i < NC; ++i) {
        const int c = warp + 32 * i;
        if (c >= p.n_chunks) break;
        float sum = 0.f, li[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = c * kC + lane * 4 + j;
            float lf = 0.f;
            li[j] = -INFINITY;
            if (t < p.T) log_gates(a.z + ((size_t)b * p.S + p.t0 + t) * a.z_ld, a.z_bias, p.H, h, a.cap, li[j], lf);
            sum += lf;
            F[i][j] = sum;
        }
        float incl = sum;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, incl, o);
            if (lane >= o) incl += v;
        }
        const float excl = incl - sum;
        float mx = -INFINITY;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            F[i][j] += excl;
            A[i][j] = li[j] - F[i][j];
            mx = fmaxf(mx, A[i][j]);
            cm[i][j] = mx;
        }
        float inclm = mx;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, inclm, o);
            if (lane >= o) inclm = fmaxf(inclm, v);
        }
        float before = __shfl_up_sync(0xffffffffu, inclm, 1);
        if (lane == 0) before = -INFINITY;
#pragma unroll
        for (int j = 0; j < 4; ++j) cm[i][j] = fmaxf(cm[i][j], before);
        if (lane == 31) {
            f_end[c] = F[i][3];
            a_max[c] = cm[i][3];
        }
    }
    __syncthreads();
    if (tid == 0) {
        float m = p.fresh ? 0.f : a.mx[bh];
        for (int c = 0; c < p.n_chunks; ++c) {
            m_0[c] = m;
            const float M = fmaxf(m, a_max[c]);
            p.decay[(size_t)bh * p.n_chunks + c] = expf(m - M);
            m = f_end[c] + M;
        }
        a.mx[bh] = m;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NC; ++i) {
        const int c = warp + 32 * i;
        if (c >= p.n_chunks) break;
        const float m0 = m_0[c], m_end = fmaxf(m0, a_max[c]);
        const size_t at = (size_t)bh * p.n_chunks * kC + c * kC + lane * 4;
        float M[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) M[j] = fmaxf(m0, cm[i][j]);
        auto put = [&](float *dst, auto f) { *reinterpret_cast<float4 *>(dst + at) = make_float4(f(0), f(1), f(2), f(3)); };
        put(p.a2, [&](int j) { return A[i][j] * kLog2e; });
        put(p.m2, [&](int j) { return M[j] * kLog2e; });
        put(p.g, [&](int j) { return expf(m0 - M[j]); });
        put(p.en, [&](int j) { return expf(-(F[i][j] + M[j])); });
        put(p.w, [&](int j) { return expf(A[i][j] - m_end); });
    }
}

// grid (chunks, column groups of 64: keys first, then values; B * H)
constexpr int kPackPitch = 66;
__global__ void __launch_bounds__(256) mlstm_pack_kernel(const Seg p) {
    __shared__ __nv_bfloat16 tile[kC][kPackPitch];
    __shared__ float ws[kC], part[4][64];
    const int tid = threadIdx.x, c = blockIdx.x, bh = blockIdx.z, b = bh / p.H, h = bh - b * p.H;
    const int kg = (p.dim + 63) / 64;
    const bool key = (int)blockIdx.y < kg;
    const int n = key ? p.dim : p.vdim, d0 = ((int)blockIdx.y - (key ? 0 : kg)) * 64, nt = min(kC, p.T - c * kC);
    const __nv_bfloat16 *src = p.u + ((size_t)b * p.S + p.t0 + c * kC) * p.u_ld + (key ? p.u_k : p.u_v) + (size_t)h * n + d0;
    if (tid < kC) ws[tid] = p.w[(size_t)bh * p.n_chunks * kC + c * kC + tid];
    for (int i = tid; i < kC * 8; i += 256) {  // 8 numbers at a time (dim, vdim and the row pitch are multiples of 8)
        const int t = i >> 3, d = (i & 7) * 8;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (t < nt && d0 + d < n) v = *reinterpret_cast<const uint4 *>(src + (size_t)t * p.u_ld + d);
        uint32_t *dst = reinterpret_cast<uint32_t *>(&tile[t][d]);
        dst[0] = v.x; dst[1] = v.y; dst[2] = v.z; dst[3] = v.w;
    }
    __syncthreads();
    const size_t pitch = (size_t)p.n_chunks * kC;
    for (int i = tid; i < 64 * (kC / 8); i += 256) {
        const int t = (i & 15) * 8, d = i >> 4;
        if (d0 + d >= n) continue;
        float x[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = __bfloat162float(tile[t + j][d]) * (key ? ws[t + j] : 1.f);
        const size_t at = ((size_t)bh * n + d0 + d) * pitch + c * kC + t;
        uint4 hi = make_uint4(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]), pack_bf16(x[4], x[5]), pack_bf16(x[6], x[7]));
        *reinterpret_cast<uint4 *>((key ? p.kt_hi : p.vt) + at) = hi;
        if (key) {
            const uint32_t *w = &hi.x;
            uint4 lo;
            uint32_t *l = &lo.x;
#pragma unroll
            for (int j = 0; j < 4; ++j) l[j] = pack_bf16(x[2 * j] - __uint_as_float(w[j] << 16), x[2 * j + 1] - __uint_as_float(w[j] & 0xffff0000u));
            *reinterpret_cast<uint4 *>(p.kt_lo + at) = lo;
        }
    }
    if (key) {
        const int d = tid & 63, q = tid >> 6;
        float s = 0.f;
#pragma unroll 8
        for (int t = q * 32; t < q * 32 + 32; ++t) s = fmaf(__bfloat162float(tile[t][d]), ws[t], s);
        part[q][d] = s;
        __syncthreads();
        if (tid < 64 && d0 + tid < p.dim)
            p.nsum[((size_t)bh * p.n_chunks + c) * p.dim + d0 + tid] = (part[0][tid] + part[1][tid]) + (part[2][tid] + part[3][tid]);
    }
}

// ---- S^T at the start of every chunk ---------------------------------------------------------------
constexpr int kStN = 64;                             // keys of a tile
constexpr uint32_t kStA = 128 * kBK * 2, kStB = kStN * kBK * 2;
constexpr uint32_t kStStage = 2 * kStA + 4 * kStB;   // v^T: two blocks of 64 tokens; weighted k^T: hi and lo of each
constexpr int kStStages = 3;
constexpr size_t kStSmem = kStStages * kStStage + 2 * kStA + 1024;  // + the tile on its way out, hi and lo

// grid (value tiles of 128, key tiles of 64, B * H); warps 0-7 keep the tile, warp 8 issues the MMAs, warp 9 the copies
__global__ void __launch_bounds__(kTcThreads, 1)
mlstm_state_kernel(const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_khi,
                   const __grid_constant__ CUtensorMap map_klo, const __grid_constant__ CUtensorMap map_shi, const __grid_constant__ CUtensorMap map_slo,
                   const Seg p) {
    extern __shared__ unsigned char smem_raw[];
    unsigned char *ring = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ uint64_t full[kStStages], empty[kStStages], d_full[2], d_free[2];
    __shared__ uint32_t tmem_base_s;
    __shared__ int failed_s;
    __shared__ float decay[kSegChunks];
    unsigned char *s_out = ring + kStStages * kStStage;
    volatile int *failed = &failed_s;
    const int tid = threadIdx.x, warp = tid >> 5, nc = p.n_chunks;
    const int m0 = blockIdx.x * 128, n0 = blockIdx.y * kStN, bh = blockIdx.z;
    if (tid == 0) {
        for (int s = 0; s < kStStages; ++s) {
            bar_init(&full[s], 1);
            bar_init(&empty[s], 1);
        }
        for (int s = 0; s < 2; ++s) {
            bar_init(&d_full[s], 1);
            bar_init(&d_free[s], kWorkers);
        }
        failed_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    for (int c = tid; c < nc; c += kTcThreads) decay[c] = p.decay[(size_t)bh * nc + c];
    if (warp == kWorkers / 32) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(saddr(&tmem_base_s)), "r"(2 * kStN) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_base_s;

    if (warp == kWorkers / 32 + 1) {
        if ((tid & 31) == 0) {
#pragma unroll 1
            for (int c = 0; c < nc; ++c) {
                const int s = c % kStStages;
                if (c >= kStStages && !wait_or_failed(&empty[s], (uint32_t)((c / kStStages - 1) & 1), failed, p.status, 700)) break;
                unsigned char *st = ring + (size_t)s * kStStage;
                bar_expect(&full[s], kStStage);
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    const int x = c * kC + k * kBK;
                    tma_load_2d(st + k * kStA, &map_v, x, bh * p.vdim + m0, &full[s]);
                    tma_load_2d(st + 2 * kStA + k * kStB, &map_khi, x, bh * p.dim + n0, &full[s]);
                    tma_load_2d(st + 2 * kStA + (2 + k) * kStB, &map_klo, x, bh * p.dim + n0, &full[s]);
                }
            }
        }
        __syncwarp();
    } else if (warp == kWorkers / 32) {
        if ((tid & 31) == 0) {
            constexpr uint32_t kIdesc = idesc_bf16(128, kStN);
#pragma unroll 1
            for (int c = 0; c < nc; ++c) {
                const int s = c % kStStages;
                bool ok = wait_or_failed(&full[s], (uint32_t)((c / kStStages) & 1), failed, p.status, 710);
                if (ok && c >= 2) ok = wait_or_failed(&d_free[c & 1], (uint32_t)(((c >> 1) - 1) & 1), failed, p.status, 711);
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (ok) {
                    const uint32_t st = saddr(ring + (size_t)s * kStStage), acc = tmem + (uint32_t)((c & 1) * kStN);
#pragma unroll
                    for (int k = 0; k < 2; ++k) {
                        const uint64_t av = smem_desc(st + k * kStA), bh_ = smem_desc(st + 2 * kStA + k * kStB), bl = smem_desc(st + 2 * kStA + (2 + k) * kStB);
#pragma unroll
                        for (int kk = 0; kk < kBK / 16; ++kk) {
                            umma_bf16(acc, av + 2 * kk, bh_ + 2 * kk, kIdesc, (k > 0 || kk > 0) ? 1u : 0u);
                            umma_bf16(acc, av + 2 * kk, bl + 2 * kk, kIdesc, 1u);
                        }
                    }
                }
                umma_commit(&empty[s]);
                umma_commit(&d_full[c & 1]);
            }
        }
        __syncwarp();
    } else {
        // thread (row, half): value m0 + row, keys n0 + 32 half ..
        const int row = tid & 127, half = tid >> 7, val = m0 + row, key0 = n0 + 32 * half;
        const uint32_t lane_off = (uint32_t)((warp & 3) * 32) << 16;
        const bool live = val < p.vdim;
        float *st = p.state + (size_t)bh * p.dim * p.vdim + val;
        float S[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) S[i] = live && !p.fresh && key0 + i < p.dim ? st[(size_t)(key0 + i) * p.vdim] : 0.f;
        // n of the tile's keys, by the CTAs of the first value tile
        const bool nlive = blockIdx.x == 0 && tid < kStN && n0 + tid < p.dim;
        float n = nlive && !p.fresh ? p.norm[(size_t)bh * p.dim + n0 + tid] : 0.f;
#pragma unroll 1
        for (int c = 0; c < nc; ++c) {
            const size_t bc = (size_t)bh * nc + c;
            if (!(p.fresh && c == 0)) {  // (the memory before the first token is not read)
                if (tid == 0) tma_store_wait_read();  // the previous chunk's copies have left shared memory
                __syncwarp();
                asm volatile("bar.sync 1, 256;" ::: "memory");
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    uint4 hi, lo;
                    uint32_t *hp = &hi.x, *lp = &lo.x;
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const float x = S[8 * q + 2 * j], y = S[8 * q + 2 * j + 1];
                        hp[j] = pack_bf16(x, y);
                        lp[j] = pack_bf16(x - __uint_as_float(hp[j] << 16), y - __uint_as_float(hp[j] & 0xffff0000u));
                    }
                    unsigned char *dst = s_out + (size_t)row * 128 + (((4 * half + q) ^ (row & 7)) << 4);  // 128-byte swizzle
                    *reinterpret_cast<uint4 *>(dst) = hi;
                    *reinterpret_cast<uint4 *>(dst + kStA) = lo;
                }
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
                asm volatile("bar.sync 1, 256;" ::: "memory");
                if (tid == 0) {
                    tma_store_3d(&map_shi, s_out, n0, m0, (int)bc);
                    tma_store_3d(&map_slo, s_out + kStA, n0, m0, (int)bc);
                    tma_store_commit();
                }
            }
            if (nlive) {
                p.nst[bc * p.dim + n0 + tid] = n;
                n = fmaf(decay[c], n, p.nsum[bc * p.dim + n0 + tid]);
            }
            wait_or_failed(&d_full[c & 1], (uint32_t)((c >> 1) & 1), failed, p.status, 720);
            __syncwarp();
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            uint32_t v[32];
            tmem_ld32(tmem + (uint32_t)((c & 1) * kStN + 32 * half) + lane_off, v);
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            bar_arrive(&d_free[c & 1]);
            const float d = decay[c];
#pragma unroll
            for (int i = 0; i < 32; ++i) S[i] = fmaf(d, S[i], __uint_as_float(v[i]));
        }
        if (live)
#pragma unroll
            for (int i = 0; i < 32; ++i)
                if (key0 + i < p.dim) st[(size_t)(key0 + i) * p.vdim] = S[i];
        if (nlive) p.norm[(size_t)bh * p.dim + n0 + tid] = n;
        if (tid == 0) tma_store_wait();
    }
    __syncthreads();
    if (*failed && tid == kWorkers + 32) {  // copies in flight land before the CTA exits (bounded)
        for (int s = 0; s < kStStages; ++s) {
            const long long t0 = clock64();
            while (!bar_try(&full[s], 0) && !bar_try(&full[s], 1) && clock64() - t0 < kTcWaitCycles) {}
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == kWorkers / 32)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(2 * kStN) : "memory");
}

// ---- outputs of a chunk -----------------------------------------------------------------------------
constexpr uint32_t kTile = 128 * kBK * 2;      // 128 rows of 128 bytes
constexpr uint32_t kOutStage = 2 * kTile;
// KB: 64-element blocks of a key
template <int KB>
struct OutGeom {
    static constexpr uint32_t kQ = KB * kTile, kP = 4 * kTile;  // weights: hi and lo of two blocks of 64 tokens
    static constexpr int kStages = (int)((226 * 1024 - kQ - kP) / kOutStage) > 4 ? 4 : (int)((226 * 1024 - kQ - kP) / kOutStage);
    static constexpr size_t kSmem = kQ + kP + kStages * kOutStage + 1024;
};

// grid (chunks, B * H, groups of value tiles).  Tensor memory, 4 regions of 128 columns: the scores in region 0; products with
// S_0 and with v of even tiles in 1 and 2, of odd ones in 3 and 0 (the scores have been read by then).
template <int KB>
__global__ void __launch_bounds__(kTcThreads, 1)
mlstm_out_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_shi,
                 const __grid_constant__ CUtensorMap map_slo, const __grid_constant__ CUtensorMap map_v, const Seg p) {
    using G = OutGeom<KB>;
    extern __shared__ unsigned char smem_raw[];
    unsigned char *q_s = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char *p_s = q_s + G::kQ, *ring = p_s + G::kP;
    __shared__ uint64_t q_bar, full[G::kStages], empty[G::kStages], s_bar, p_bar, o_full[2], o_free[2];
    __shared__ uint32_t tmem_base_s;
    __shared__ int failed_s;
    __shared__ float a2_s[kC], xch[2][kC];
    volatile int *failed = &failed_s;
    const int tid = threadIdx.x, warp = tid >> 5;
    const int c = blockIdx.x, bh = blockIdx.y, b = bh / p.H, h = bh - b * p.H;
    const int per = (p.tiles + (int)gridDim.z - 1) / (int)gridDim.z, j0 = (int)blockIdx.z * per, nj = min(p.tiles, j0 + per) - j0;
    const bool has_prev = !(p.fresh && c == 0);
    const size_t bc = (size_t)bh * p.n_chunks + c, tok = (size_t)bh * p.n_chunks * kC + c * kC;
    if (nj <= 0) return;  // (the same for the whole CTA, before anything is set up)
    if (tid == 0) {
        bar_init(&q_bar, 1);
        for (int s = 0; s < G::kStages; ++s) {
            bar_init(&full[s], 1);
            bar_init(&empty[s], 1);
        }
        bar_init(&s_bar, 1);
        bar_init(&p_bar, kWorkers);
        for (int s = 0; s < 2; ++s) {
            bar_init(&o_full[s], 1);
            bar_init(&o_free[s], kWorkers);
        }
        failed_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    for (int i = tid; i < kC; i += kTcThreads) a2_s[i] = p.a2[tok + i];
    if (warp == kWorkers / 32) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(saddr(&tmem_base_s)), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_base_s;
    auto inter_cols = [&](int j) { return tmem + ((j & 1) ? 3u : 1u) * 128u; };
    auto intra_cols = [&](int j) { return tmem + ((j & 1) ? 0u : 2u) * 128u; };

    if (warp == kWorkers / 32 + 1) {
        if ((tid & 31) == 0) {
            const int row0 = b * p.S + p.t0 + c * kC;
            int it = 0;
            // a free stage, announced with its bytes
            auto next = [&](uint32_t bytes) -> unsigned char * {
                const int s = it % G::kStages;
                if (it >= G::kStages && !wait_or_failed(&empty[s], (uint32_t)((it / G::kStages - 1) & 1), failed, p.status, 740)) return nullptr;
                bar_expect(&full[s], bytes);
                return ring + (size_t)s * kOutStage;
            };
            bar_expect(&q_bar, G::kQ);
#pragma unroll
            for (int kb = 0; kb < KB; ++kb) tma_load_3d(q_s + kb * kTile, &map_q, kb * kBK, h, row0, &q_bar);
#pragma unroll 1
            for (int kb = 0; kb < KB; ++kb, ++it) {
                unsigned char *st = next(kTile);
                if (!st) break;
                tma_load_3d(st, &map_k, kb * kBK, h, row0, &full[it % G::kStages]);
            }
#pragma unroll 1
            for (int j = 0; j < nj && !*failed; ++j) {
                const int d0 = (j0 + j) * 128;
                if (has_prev)
#pragma unroll 1
                    for (int kb = 0; kb < KB; ++kb, ++it) {
                        unsigned char *st = next(2 * kTile);
                        if (!st) break;
                        const int y = (int)(bc * p.vdim) + d0;
                        tma_load_2d(st, &map_shi, kb * kBK, y, &full[it % G::kStages]);
                        tma_load_2d(st + kTile, &map_slo, kb * kBK, y, &full[it % G::kStages]);
                    }
                unsigned char *st = next(2 * kTile);
                if (!st) break;
#pragma unroll
                for (int k = 0; k < 2; ++k) tma_load_2d(st + k * kTile, &map_v, c * kC + k * kBK, bh * p.vdim + d0, &full[it % G::kStages]);
                ++it;
            }
        }
        __syncwarp();
    } else if (warp == kWorkers / 32) {
        if ((tid & 31) == 0) {
            constexpr uint32_t kIdesc = idesc_bf16(128, 128);
            int it = 0;
            const uint32_t qa = saddr(q_s), pa = saddr(p_s);
            auto stage_ready = [&](int site) {
                const int s = it % G::kStages;
                const bool ok = wait_or_failed(&full[s], (uint32_t)((it / G::kStages) & 1), failed, p.status, site);
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                return ok;
            };
            wait_or_failed(&q_bar, 0, failed, p.status, 750);
#pragma unroll 1
            for (int kb = 0; kb < KB; ++kb, ++it) {
                const int s = it % G::kStages;
                if (stage_ready(751)) {
                    const uint64_t q = smem_desc(qa + kb * kTile), k = smem_desc(saddr(ring + (size_t)s * kOutStage));
#pragma unroll
                    for (int kk = 0; kk < kBK / 16; ++kk) umma_bf16(tmem, q + 2 * kk, k + 2 * kk, kIdesc, (kb > 0 || kk > 0) ? 1u : 0u);
                }
                umma_commit(&empty[s]);
            }
            umma_commit(&s_bar);
#pragma unroll 1
            for (int j = 0; j < nj; ++j) {
                if (j >= 2) wait_or_failed(&o_free[j & 1], (uint32_t)(((j >> 1) - 1) & 1), failed, p.status, 752);
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (has_prev)
#pragma unroll 1
                    for (int kb = 0; kb < KB; ++kb, ++it) {
                        const int s = it % G::kStages;
                        if (stage_ready(753)) {
                            const uint32_t st = saddr(ring + (size_t)s * kOutStage);
                            const uint64_t q = smem_desc(qa + kb * kTile), hi = smem_desc(st), lo = smem_desc(st + kTile);
#pragma unroll
                            for (int kk = 0; kk < kBK / 16; ++kk) {
                                umma_bf16(inter_cols(j), q + 2 * kk, hi + 2 * kk, kIdesc, (kb > 0 || kk > 0) ? 1u : 0u);
                                umma_bf16(inter_cols(j), q + 2 * kk, lo + 2 * kk, kIdesc, 1u);
                            }
                        }
                        umma_commit(&empty[s]);
                    }
                if (j == 0) wait_or_failed(&p_bar, 0, failed, p.status, 754);
                const int s = it % G::kStages;
                if (stage_ready(755)) {
                    const uint32_t st = saddr(ring + (size_t)s * kOutStage);
#pragma unroll
                    for (int k = 0; k < 2; ++k) {
                        const uint64_t hi = smem_desc(pa + k * kTile), lo = smem_desc(pa + (2 + k) * kTile), v = smem_desc(st + k * kTile);
#pragma unroll
                        for (int kk = 0; kk < kBK / 16; ++kk) {
                            umma_bf16(intra_cols(j), hi + 2 * kk, v + 2 * kk, kIdesc, (k > 0 || kk > 0) ? 1u : 0u);
                            umma_bf16(intra_cols(j), lo + 2 * kk, v + 2 * kk, kIdesc, 1u);
                        }
                    }
                }
                umma_commit(&empty[s]);
                umma_commit(&o_full[j & 1]);
                ++it;
            }
        }
        __syncwarp();
    } else {
        // thread (row, half): token `row` of the chunk; 64 of its 128 scores, 64 of every 128 values
        const int row = tid & (kC - 1), half = tid >> 7, quad = warp & 3;
        const uint32_t lane_off = (uint32_t)(quad * 32) << 16;
        const float m2 = p.m2[tok + row], g = p.g[tok + row], en = p.en[tok + row];
        wait_or_failed(&s_bar, 0, failed, p.status, 760);
        __syncwarp();
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        float sum = 0.f;
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            uint32_t v[32], hi[16], lo[16];
            tmem_ld32(tmem + lane_off + 64 * half + 32 * q, v);
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                float w[2];
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    const int s = 64 * half + 32 * q + 2 * i + k;
                    w[k] = s <= row ? __uint_as_float(v[2 * i + k]) * p.qscale * ex2(a2_s[s] - m2) : 0.f;
                    sum += w[k];
                }
                hi[i] = pack_bf16(w[0], w[1]);
                lo[i] = pack_bf16(w[0] - __uint_as_float(hi[i] << 16), w[1] - __uint_as_float(hi[i] & 0xffff0000u));
            }
            unsigned char *prow = p_s + half * kTile + (size_t)row * 128;
#pragma unroll
            for (int c8 = 0; c8 < 4; ++c8) {
                const int off = ((4 * q + c8) ^ (row & 7)) << 4;  // 128-byte swizzle
                *reinterpret_cast<uint4 *>(prow + off) = make_uint4(hi[4 * c8], hi[4 * c8 + 1], hi[4 * c8 + 2], hi[4 * c8 + 3]);
                *reinterpret_cast<uint4 *>(prow + 2 * kTile + off) = make_uint4(lo[4 * c8], lo[4 * c8 + 1], lo[4 * c8 + 2], lo[4 * c8 + 3]);
            }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
        bar_arrive(&p_bar);
        if (has_prev) {  // n_0 . q: this half's share of every block
            wait_or_failed(&q_bar, 0, failed, p.status, 761);
            float dot = 0.f;
#pragma unroll
            for (int kb = 0; kb < KB; ++kb)
#pragma unroll
                for (int c8 = 0; c8 < 4; ++c8) {
                    const int ch = 4 * half + c8;
                    if (kb * kBK + ch * 8 >= p.dim) continue;  // (dim is a multiple of 8)
                    const uint4 v = *reinterpret_cast<const uint4 *>(q_s + kb * kTile + (size_t)row * 128 + ((ch ^ (row & 7)) << 4));
                    const float4 *n4 = reinterpret_cast<const float4 *>(p.nst + bc * p.dim + kb * kBK + ch * 8);  // the same for the warp
                    const float4 na = __ldg(n4), nb = __ldg(n4 + 1);
                    dot = fmaf(__uint_as_float(v.x << 16), na.x, fmaf(__uint_as_float(v.x & 0xffff0000u), na.y, dot));
                    dot = fmaf(__uint_as_float(v.y << 16), na.z, fmaf(__uint_as_float(v.y & 0xffff0000u), na.w, dot));
                    dot = fmaf(__uint_as_float(v.z << 16), nb.x, fmaf(__uint_as_float(v.z & 0xffff0000u), nb.y, dot));
                    dot = fmaf(__uint_as_float(v.w << 16), nb.z, fmaf(__uint_as_float(v.w & 0xffff0000u), nb.w, dot));
                }
            sum = fmaf(g * p.qscale, dot, sum);
        }
        xch[half][row] = sum;
        asm volatile("bar.sync %0, 64;" ::"r"(1 + quad) : "memory");  // the row's other half: warp w ^ 4
        const float rden = __fdiv_rn(1.0f, fmaxf(fabsf(xch[0][row] + xch[1][row]), en) + 1e-6f);
        const float gq = g * p.qscale;
        const int t = c * kC + row;
        const bool live = t < p.T;
        const size_t orow = ((size_t)b * p.T + t) * p.H + h;
#pragma unroll 1
        for (int j = 0; j < nj; ++j) {
            wait_or_failed(&o_full[j & 1], (uint32_t)((j >> 1) & 1), failed, p.status, 762);
            __syncwarp();
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            float ssq = 0.f;
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                uint32_t x[32], y[32];
                const uint32_t off = lane_off + 64 * half + 32 * q;
                tmem_ld32_issue(intra_cols(j) + off, x);
                if (has_prev) tmem_ld32_issue(inter_cols(j) + off, y);
                tmem_ld_wait();
                const int col = (j0 + j) * 128 + 64 * half + 32 * q;
                uint32_t r[16];
#pragma unroll
                for (int i = 0; i < 32; i += 2) {
                    float o0 = __uint_as_float(x[i]), o1 = __uint_as_float(x[i + 1]);
                    if (has_prev) {
                        o0 = fmaf(gq, __uint_as_float(y[i]), o0);
                        o1 = fmaf(gq, __uint_as_float(y[i + 1]), o1);
                    }
                    o0 *= rden;
                    o1 *= rden;
                    if (col + i < p.vdim) ssq = fmaf(o0, o0, fmaf(o1, o1, ssq));  // (vdim is even)
                    r[i / 2] = pack_bf16(o0, o1);
                }
                if (live)
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (col + 8 * i < p.vdim)
                            *reinterpret_cast<uint4 *>(p.o + orow * p.vdim + col + 8 * i) = make_uint4(r[4 * i], r[4 * i + 1], r[4 * i + 2], r[4 * i + 3]);
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            bar_arrive(&o_free[j & 1]);
            if (live) p.ssq[(orow * p.tiles + j0 + j) * 2 + half] = ssq;
        }
    }
    __syncthreads();
    if (*failed && tid == kWorkers + 32) {  // copies in flight land before the CTA exits (bounded)
        const long long t0 = clock64();
        while (!bar_try(&q_bar, 0) && clock64() - t0 < kTcWaitCycles) {}
        for (int s = 0; s < G::kStages; ++s) {
            const long long t1 = clock64();
            while (!bar_try(&full[s], 0) && !bar_try(&full[s], 1) && clock64() - t1 < kTcWaitCycles) {}
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == kWorkers / 32) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512) : "memory");
}

// One thread per 8 outputs of a row.
__global__ void __launch_bounds__(256) mlstm_finish_kernel(const Seg p, const float *__restrict__ gain, float eps, float *__restrict__ out,
                                                           __nv_bfloat16 *__restrict__ hi, __nv_bfloat16 *__restrict__ lo) {
    const unsigned i = blockIdx.x * 256 + threadIdx.x, per_row = (unsigned)p.H * p.vdim / 8, row = i / per_row;  // (see mlstm_chunked_usable)
    if (row >= (unsigned)(p.B * p.T)) return;
    const unsigned j = (i - row * per_row) * 8, h = j / (unsigned)p.vdim, b = row / (unsigned)p.T;
    const size_t m = (size_t)b * p.S + p.t0 + (row - b * p.T);
    const float *ss = p.ssq + ((size_t)row * p.H + h) * 2 * p.tiles;
    float s = 0.f;
    for (int k = 0; k < 2 * p.tiles; ++k) s += ss[k];
    const float inv = __fdiv_rn(1.0f, sqrtf(__fadd_rn(__fdiv_rn(s, (float)p.vdim), eps)));
    const uint4 ov = *reinterpret_cast<const uint4 *>(p.o + (size_t)i * 8), gv = *reinterpret_cast<const uint4 *>(p.u + m * p.u_ld + p.u_g + j);
    const float4 n0 = *reinterpret_cast<const float4 *>(gain + j), n1 = *reinterpret_cast<const float4 *>(gain + j + 4);
    const float n[8] = {n0.x, n0.y, n0.z, n0.w, n1.x, n1.y, n1.z, n1.w};
    const uint32_t *ow = &ov.x, *gw = &gv.x;
    const size_t at = m * (size_t)p.H * p.vdim + j;
    float v[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
        const float o = __uint_as_float(k & 1 ? ow[k / 2] & 0xffff0000u : ow[k / 2] << 16), g = __uint_as_float(k & 1 ? gw[k / 2] & 0xffff0000u : gw[k / 2] << 16);
        v[k] = o * inv * n[k] * __fdividef(1.0f, 1.0f + ex2(-g * kLog2e));  // (rounded to 16 bits next; 1 / inf = 0)
    }
    if (hi && !lo) {
        *reinterpret_cast<uint4 *>(hi + at) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
    } else if (hi) {
#pragma unroll
        for (int k = 0; k < 8; ++k) store_split(v[k], hi, lo, at + k);
    }
    if (out)
#pragma unroll
        for (int k = 0; k < 8; ++k) out[at + k] = v[k];
}

template <int KB>
int launch_out(lumen_ctx *ctx, const CUtensorMap *maps, const Seg &p, dim3 grid, cudaStream_t s) {
    using G = OutGeom<KB>;
    LUMEN_CUDA(ctx, cudaFuncSetAttribute(mlstm_out_kernel<KB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)G::kSmem));
    mlstm_out_kernel<KB><<<grid, kTcThreads, G::kSmem, s>>>(maps[0], maps[1], maps[2], maps[3], maps[4], p);
    LUMEN_LAUNCHED(ctx);
    return LUMEN_OK;
}

}  // namespace

// Portions of at least 64 tokens, keys of at most 256 numbers, 16-byte steps between heads and rows.
bool mlstm_chunked_usable(const MlstmArgs &a) {
    static const bool off = [] {
        const char *e = getenv("LUMEN_NO_TC_ATTN");
        return e && e[0] == '1';
    }();
    return !off && a.S >= 64 && a.dim <= 256 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.u_ld % 8 == 0 && a.B * a.H <= 65535 &&
           a.B * a.S * a.H * a.vdim / 8 < ((size_t)1 << 31) && a.B * a.S < ((size_t)1 << 31) && a.B * a.H * kSegChunks * std::max(a.vdim, a.dim) < ((size_t)1 << 31);
}

int launch_mlstm_chunked(lumen_ctx *ctx, const MlstmArgs &a, cudaStream_t s) {
    const size_t BH = a.B * a.H, seg_T = std::min<size_t>(a.S, (size_t)kSegChunks * kC), nc = (seg_T + kC - 1) / kC, tp = nc * kC;
    const size_t tiles = (a.vdim + 127) / 128;
    size_t off = 0;
    auto take = [&](size_t bytes) { const size_t o = off; off += (bytes + 255) / 256 * 256; return o; };
    const size_t o_a2 = take(BH * tp * 4), o_m2 = take(BH * tp * 4), o_g = take(BH * tp * 4), o_en = take(BH * tp * 4), o_w = take(BH * tp * 4),
                 o_dec = take(BH * nc * 4), o_kh = take(BH * a.dim * tp * 2), o_kl = take(BH * a.dim * tp * 2), o_vt = take(BH * a.vdim * tp * 2),
                 o_ns = take(BH * nc * a.dim * 4), o_nt = take(BH * nc * a.dim * 4), o_sh = take(BH * nc * a.vdim * a.dim * 2),
                 o_sl = take(BH * nc * a.vdim * a.dim * 2), o_o = take(a.B * seg_T * a.H * a.vdim * 2), o_ss = take(a.B * seg_T * a.H * 2 * tiles * 4);
    void *ws = nullptr;
    LUMEN_TRY(dev_alloc(ctx, off, &ws));
    char *base = static_cast<char *>(ws);
    auto f = [&](size_t o) { return reinterpret_cast<float *>(base + o); };
    auto bf = [&](size_t o) { return reinterpret_cast<__nv_bfloat16 *>(base + o); };
    Seg p{};
    p.B = (int)a.B; p.S = (int)a.S; p.H = (int)a.H; p.dim = (int)a.dim; p.vdim = (int)a.vdim;
    p.u = a.u16; p.u_ld = a.u_ld; p.u_k = a.u_k; p.u_v = a.u_v; p.u_g = a.u_g;
    p.a2 = f(o_a2); p.m2 = f(o_m2); p.g = f(o_g); p.en = f(o_en); p.w = f(o_w); p.decay = f(o_dec);
    p.kt_hi = bf(o_kh); p.kt_lo = bf(o_kl); p.vt = bf(o_vt); p.nsum = f(o_ns); p.nst = f(o_nt); p.s_hi = bf(o_sh); p.s_lo = bf(o_sl);
    p.state = a.state; p.norm = a.norm; p.o = bf(o_o); p.ssq = f(o_ss); p.tiles = (int)tiles;
    p.qscale = 1.0f / sqrtf((float)a.dim); p.status = ctx->d_status;
    auto segment = [&]() -> int {
        const unsigned c = (unsigned)p.n_chunks, kg = (unsigned)((a.dim + 63) / 64), vg = (unsigned)((a.vdim + 63) / 64);
        mlstm_scan_kernel<<<(unsigned)BH, 1024, 0, s>>>(a, p);
        LUMEN_LAUNCHED(ctx);
        mlstm_pack_kernel<<<dim3(c, kg + vg, (unsigned)BH), 256, 0, s>>>(p);
        LUMEN_LAUNCHED(ctx);
        const size_t pitch = (size_t)c * kC;
        CUtensorMap st[5], out[5];
        LUMEN_TRY(make_map(ctx, &st[0], p.vt, BH * a.vdim, pitch, 128));
        LUMEN_TRY(make_map(ctx, &st[1], p.kt_hi, BH * a.dim, pitch, kStN));
        LUMEN_TRY(make_map(ctx, &st[2], p.kt_lo, BH * a.dim, pitch, kStN));
        LUMEN_TRY(make_map_3d(ctx, &st[3], p.s_hi, a.dim, a.vdim, a.dim, BH * c, a.vdim * a.dim, 128, 1));
        LUMEN_TRY(make_map_3d(ctx, &st[4], p.s_lo, a.dim, a.vdim, a.dim, BH * c, a.vdim * a.dim, 128, 1));
        LUMEN_CUDA(ctx, cudaFuncSetAttribute(mlstm_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kStSmem));
        mlstm_state_kernel<<<dim3((unsigned)tiles, kg, (unsigned)BH), kTcThreads, kStSmem, s>>>(st[0], st[1], st[2], st[3], st[4], p);
        LUMEN_LAUNCHED(ctx);
        LUMEN_TRY(make_map_3d(ctx, &out[0], a.u16, a.dim, a.H, a.dim, a.B * a.S, a.u_ld, 1, kC));
        LUMEN_TRY(make_map_3d(ctx, &out[1], a.u16 + a.u_k, a.dim, a.H, a.dim, a.B * a.S, a.u_ld, 1, kC));
        LUMEN_TRY(make_map(ctx, &out[2], p.s_hi, BH * c * a.vdim, a.dim, 128));
        LUMEN_TRY(make_map(ctx, &out[3], p.s_lo, BH * c * a.vdim, a.dim, 128));
        out[4] = st[0];
        // as many groups of value tiles as the device holds at a time (scores are computed once per group)
        const unsigned z = (unsigned)std::max<size_t>(1, std::min<size_t>(tiles, ctx->num_sms / (c * BH)));
        const dim3 grid(c, (unsigned)BH, z);
        switch ((a.dim + kBK - 1) / kBK) {
            case 1: LUMEN_TRY(launch_out<1>(ctx, out, p, grid, s)); break;
            case 2: LUMEN_TRY(launch_out<2>(ctx, out, p, grid, s)); break;
            case 3: LUMEN_TRY(launch_out<3>(ctx, out, p, grid, s)); break;
            default: LUMEN_TRY(launch_out<4>(ctx, out, p, grid, s));
        }
        const size_t n = a.B * p.T * a.H * a.vdim / 8;
        mlstm_finish_kernel<<<(unsigned)((n + 255) / 256), 256, 0, s>>>(p, a.head_gain, a.eps, a.out, a.out_hi, a.out_lo);
        LUMEN_LAUNCHED(ctx);
        return LUMEN_OK;
    };
    int rc = LUMEN_OK;
    for (size_t t0 = 0; t0 < a.S && rc == LUMEN_OK; t0 += seg_T) {
        p.t0 = (int)t0;
        p.T = (int)std::min(seg_T, a.S - t0);
        p.n_chunks = (p.T + kC - 1) / kC;
        p.fresh = a.past + t0 == 0;
        rc = segment();
    }
    const int rc2 = dev_free(ctx, ws);
    return rc != LUMEN_OK ? rc : rc2;
}

}  // namespace lumen
