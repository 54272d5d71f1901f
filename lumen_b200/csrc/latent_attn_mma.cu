// Latent attention of few query positions (decode, short portions) over a bf16 cache: every head reads the same cached rows,
// so the query rows (position, head) of a sequence form the M side of a matrix product and a tile of cached rows, brought
// to shared memory once, serves all of them, first as keys (whole rows) and then as values (the latent part).
//
// A CTA takes 16 or 32 query rows and one piece of the context, 64 cached rows at a time (double buffered, cp.async).  Eight
// warps: warp w multiplies the query rows with cached rows 8 w .. 8 w + 7 (mma m16n8k16, f32 accumulators), the scores
// meet in shared memory for the running softmax, and warp w accumulates columns 8 NT w .. of the weighted latents.  The
// tensor pipe is nearly idle here - the kernel streams the cache - and 16 query rows would fill an eighth of a tcgen05
// tile.  Softmax weights enter the second product as a bf16 hi/lo pair.
#include <algorithm>

#include "decoder_kernels.cuh"
#include "mma_common.cuh"

namespace lumen {
namespace {

constexpr int kWarps = 8, kThreads = kWarps * 32;
constexpr int kBN = kLatentTile;   // cached rows per tile
constexpr int kLdS = kBN + 4;      // floats between score rows
constexpr int kLdP = kBN + 8;      // bf16 between weight rows (16 bytes more than a multiple of 128)

__device__ __forceinline__ uint32_t saddr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp16(void *dst, const void *src, bool valid) {
    const int n = valid ? 16 : 0;  // zero-filled otherwise
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(saddr(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
struct MmaGeom {
    size_t q, k, s, p, stats, total;
};
__host__ __device__ inline MmaGeom mma_geom(int rows, int pitch) {
    MmaGeom g;
    const size_t ld = (size_t)(pitch + 8) * 2;  // an odd number of 16-byte units: ldmatrix rows fall into different banks
    g.q = 0;
    g.k = g.q + rows * ld;
    g.s = g.k + 2 * kBN * ld;
    g.p = g.s + (size_t)rows * kLdS * 4;
    g.stats = g.p + 2 * (size_t)rows * kLdP * 2;
    g.total = g.stats + (size_t)rows * 3 * 4;
    return g;
}

// grid (pieces, blocks of MT * 16 query rows, batch rows)
template <int MT, int NT>
__global__ void __launch_bounds__(kThreads, 1) latent_attn_mma_kernel(const LatentArgs a) {
    constexpr int kRows = MT * 16;
    extern __shared__ __align__(16) unsigned char smem[];
    const int pitch = (int)a.pitch, rank = (int)a.rank, ld = pitch + 8;
    const MmaGeom g = mma_geom(kRows, pitch);
    __nv_bfloat16 *qs = reinterpret_cast<__nv_bfloat16 *>(smem + g.q);
    __nv_bfloat16 *ks = reinterpret_cast<__nv_bfloat16 *>(smem + g.k);
    float *sc = reinterpret_cast<float *>(smem + g.s);
    __nv_bfloat16 *ph = reinterpret_cast<__nv_bfloat16 *>(smem + g.p), *pl = ph + kRows * kLdP;
    float *m_s = reinterpret_cast<float *>(smem + g.stats), *l_s = m_s + kRows, *f_s = l_s + kRows;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    pdl_wait();
    pdl_launch();
    const int H = (int)a.H, n_rows = (int)(a.S * a.H), row0 = blockIdx.y * kRows, b = blockIdx.z, split = blockIdx.x;
    const int past = *a.d_len, total = past + (int)a.S;
    const int pieces = latent_pieces(total, a.nsplit);  // later pieces are empty, and not read by the merge
    if (split >= pieces) return;
    // the last query row of this block sees up to past + its position
    const int seen = past + min(row0 + kRows - 1, n_rows - 1) / H + 1;
    const int j0 = latent_piece_start(total, pieces, split), j1 = min(seen, latent_piece_start(total, pieces, split + 1));
    const int nt = j1 > j0 ? (j1 - j0 + kBN - 1) / kBN : 0;
    const __nv_bfloat16 *cache = static_cast<const __nv_bfloat16 *>(a.cache) + (size_t)b * a.max_seq * pitch;
    const int vec = pitch / 8;

    auto load_tile = [&](int t) {
        __nv_bfloat16 *dst = ks + (size_t)(t & 1) * kBN * ld;
        const int base = j0 + t * kBN;
        for (int i = tid; i < kBN * vec; i += kThreads) {
            const int r = i / vec, c = i - r * vec, j = base + r;
            const bool ok = j < j1;
            cp16(dst + r * ld + c * 8, cache + (size_t)(ok ? j : base) * pitch + c * 8, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (nt > 0) {
        const __nv_bfloat16 *q = static_cast<const __nv_bfloat16 *>(a.qf) + (size_t)b * n_rows * pitch;
        for (int i = tid; i < kRows * vec; i += kThreads) {
            const int r = i / vec, c = i - r * vec;
            const bool ok = row0 + r < n_rows;
            cp16(qs + r * ld + c * 8, q + (size_t)(ok ? row0 + r : row0) * pitch + c * 8, ok);
        }
        load_tile(0);  // (the first group also holds Q)
    }
    if (tid < kRows) {
        m_s[tid] = -INFINITY;
        l_s[tid] = 0.f;
    }
    float acc[MT][NT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[mt][n][i] = 0.f;
    const int ksteps = pitch / 16;
    // softmax: 256 / kRows threads share a row
    constexpr int kPer = kThreads / kRows, kCols = kBN / kPer;
    const int srow = tid / kPer, sc0 = (tid % kPer) * kCols;
    const int s_last = row0 + srow < n_rows ? past + (row0 + srow) / H : -1;  // last cached row this query row sees

#pragma unroll 1
    for (int t = 0; t < nt; ++t) {
        if (t + 1 < nt) {
            load_tile(t + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const __nv_bfloat16 *kt = ks + (size_t)(t & 1) * kBN * ld;
        {  // scores of cached rows 8 * warp .. + 7; four chains of accumulators
            float s[MT][4][4];
#pragma unroll
            for (int mt = 0; mt < MT; ++mt)
#pragma unroll
                for (int c = 0; c < 4; ++c)
#pragma unroll
                    for (int i = 0; i < 4; ++i) s[mt][c][i] = 0.f;
            // A: rows lane % 16, halves of 8 columns by lane / 16.  B (two k steps at once): rows lane % 8, 8-column groups by lane / 8.
            const uint32_t qa = saddr(qs + (lane & 15) * ld + (lane >> 4) * 8);
            const uint32_t kb = saddr(kt + (warp * 8 + (lane & 7)) * ld + (lane >> 3) * 8);
            auto two_steps = [&](int k, int chain) {
                uint32_t bf[4];
                ldsm4(bf, kb + k * 32);
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    uint32_t af[4];
                    ldsm4(af, qa + mt * 16 * ld * 2 + k * 32);
                    mma16816(s[mt][chain], af, bf[0], bf[1]);
                    ldsm4(af, qa + mt * 16 * ld * 2 + k * 32 + 32);
                    mma16816(s[mt][chain + 1], af, bf[2], bf[3]);
                }
            };
            int k = 0;
#pragma unroll 2
            for (; k + 3 < ksteps; k += 4) {
                two_steps(k, 0);
                two_steps(k + 2, 2);
            }
            if (k + 1 < ksteps) {
                two_steps(k, 0);
                k += 2;
            }
            if (k < ksteps) {  // odd number of k steps: the rows' 8 elements of padding are read but not used
                uint32_t bf[4];
                ldsm4(bf, saddr(kt + (warp * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8) + k * 32);
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    uint32_t af[4];
                    ldsm4(af, qa + mt * 16 * ld * 2 + k * 32);
                    mma16816(s[mt][0], af, bf[0], bf[1]);
                }
            }
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                float *o = sc + (mt * 16 + (lane >> 2)) * kLdS + warp * 8 + (lane & 3) * 2;
                o[0] = (s[mt][0][0] + s[mt][1][0]) + (s[mt][2][0] + s[mt][3][0]);
                o[1] = (s[mt][0][1] + s[mt][1][1]) + (s[mt][2][1] + s[mt][3][1]);
                o[8 * kLdS] = (s[mt][0][2] + s[mt][1][2]) + (s[mt][2][2] + s[mt][3][2]);
                o[8 * kLdS + 1] = (s[mt][0][3] + s[mt][1][3]) + (s[mt][2][3] + s[mt][3][3]);
            }
        }
        __syncthreads();
        {  // running softmax
            const int key0 = j0 + t * kBN + sc0, lim = min(s_last, j1 - 1);
            float v[kCols], mx = -INFINITY;
#pragma unroll
            for (int c = 0; c < kCols; ++c) {
                v[c] = key0 + c <= lim ? sc[srow * kLdS + sc0 + c] * a.scale : -INFINITY;
                mx = fmaxf(mx, v[c]);
            }
#pragma unroll
            for (int o = kPer / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float m_old = m_s[srow], mn = fmaxf(m_old, mx);
            float sum = 0.f;
#pragma unroll
            for (int c = 0; c < kCols; c += 2) {
                const float w0 = mn == -INFINITY ? 0.f : expf(v[c] - mn), w1 = mn == -INFINITY ? 0.f : expf(v[c + 1] - mn);
                sum += w0 + w1;
                const __nv_bfloat162 h = __floats2bfloat162_rn(w0, w1);
                const __nv_bfloat162 l = __floats2bfloat162_rn(w0 - __low2float(h), w1 - __high2float(h));
                *reinterpret_cast<__nv_bfloat162 *>(ph + srow * kLdP + sc0 + c) = h;
                *reinterpret_cast<__nv_bfloat162 *>(pl + srow * kLdP + sc0 + c) = l;
            }
#pragma unroll
            for (int o = kPer / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            if (tid % kPer == 0) {
                const float r = mn == -INFINITY ? 1.f : expf(m_old - mn);
                m_s[srow] = mn;
                l_s[srow] = fmaf(l_s[srow], r, sum);
                f_s[srow] = r;
            }
        }
        __syncthreads();
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
            const float r0 = f_s[mt * 16 + (lane >> 2)], r1 = f_s[mt * 16 + (lane >> 2) + 8];
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                acc[mt][n][0] *= r0; acc[mt][n][1] *= r0;
                acc[mt][n][2] *= r1; acc[mt][n][3] *= r1;
            }
        }
#pragma unroll
        for (int kk = 0; kk < kBN / 16; kk += 2) {  // two k steps: one transposed load brings both B fragments of a column group
            uint32_t ah[MT][2][4], al[MT][2][4];
#pragma unroll
            for (int mt = 0; mt < MT; ++mt)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int off = (mt * 16 + (lane & 15)) * kLdP + (kk + i) * 16 + (lane >> 4) * 8;
                    ldsm4(ah[mt][i], saddr(ph + off));
                    ldsm4(al[mt][i], saddr(pl + off));
                }
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                const int col = (warp * NT + n) * 8;
                if (col < rank) {
                    uint32_t bf[4];
                    ldsm4_t(bf, saddr(kt + (kk * 16 + lane) * ld + col));
#pragma unroll
                    for (int mt = 0; mt < MT; ++mt) {
                        mma16816(acc[mt][n], ah[mt][0], bf[0], bf[1]);
                        mma16816(acc[mt][n], al[mt][0], bf[0], bf[1]);
                        mma16816(acc[mt][n], ah[mt][1], bf[2], bf[3]);
                        mma16816(acc[mt][n], al[mt][1], bf[2], bf[3]);
                    }
                }
            }
        }
        __syncthreads();  // the tile's buffer is refilled, and the weights rewritten, in the next iteration
    }
    __syncthreads();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = row0 + mt * 16 + (lane >> 2) + (i >> 1) * 8;
            if (r >= n_rows) continue;
            float *o = a.part_ctx + (((size_t)b * n_rows + r) * a.nsplit + split) * rank;
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                const int col = (warp * NT + n) * 8 + (lane & 3) * 2 + (i & 1);
                if (col < rank) o[col] = acc[mt][n][i];
            }
        }
    if (tid < kRows && row0 + tid < n_rows) {
        float *o = a.part_ml + (((size_t)b * n_rows + row0 + tid) * a.nsplit + split) * 2;
        o[0] = m_s[tid];
        o[1] = l_s[tid];
    }
}

template <int MT, int NT>
int launch_t(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s) {
    const size_t smem = mma_geom(MT * 16, (int)a.pitch).total;
    static size_t set[64] = {0};
    const int dev = ctx->device >= 0 && ctx->device < 64 ? ctx->device : 0;
    if (smem > set[dev]) {
        LUMEN_CUDA(ctx, cudaFuncSetAttribute(latent_attn_mma_kernel<MT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        set[dev] = smem;
    }
    const size_t rows = a.S * a.H;
    return launch_pdl(ctx, latent_attn_mma_kernel<MT, NT>, dim3((unsigned)a.nsplit, (unsigned)((rows + MT * 16 - 1) / (MT * 16)), (unsigned)a.B), kThreads,
                      smem, s, a);
}

constexpr size_t kSmemLimit = 227 * 1024;
int row_tiles(const LatentArgs &a) { return a.S * a.H > 16 && mma_geom(32, (int)a.pitch).total <= kSmemLimit ? 2 : 1; }

}  // namespace

bool latent_mma_usable(const LatentArgs &a) {
    static const bool off = [] {
        const char *e = getenv("LUMEN_NO_LATENT_MMA");
        return e && e[0] == '1';
    }();
    return !off && a.dt == LUMEN_BF16 && a.pitch % 16 == 0 && a.rank <= 512 && mma_geom(16, (int)a.pitch).total <= kSmemLimit && a.B <= 65535 &&
           a.S * a.H <= 16 * 65535;
}

constexpr int kMaxPieces = 128;
// Pieces of the context: about one CTA per SM over query-row blocks and batch rows; powers of two so that a handful of captured
// graphs covers every context length (with fewer tiles than pieces the last pieces stay empty).
int latent_pick_splits(const LatentArgs &a, size_t total, int num_sms) {
    const bool mma = latent_mma_usable(a);
    const size_t rows = a.S * a.H, blocks = a.B * (mma ? (rows + row_tiles(a) * 16 - 1) / (row_tiles(a) * 16) : rows);
    const size_t want = std::min<size_t>({(total + kBN - 1) / kBN, std::max<size_t>(1, (size_t)num_sms * (mma ? 1 : 8) / std::max<size_t>(blocks, 1)), (size_t)kMaxPieces});
    int n = 1;
    while ((size_t)n < want) n <<= 1;
    return std::min(n, kMaxPieces);
}

int launch_latent_mma(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s) {
    if (!latent_mma_usable(a)) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "latent attention: rank %zu, pitch %zu", a.rank, a.pitch);
    const int mt = row_tiles(a);
    const size_t groups = (a.rank + 63) / 64;  // column groups of 8 per warp
#define LUMEN_MMA(NT_) (mt == 2 ? launch_t<2, NT_>(ctx, a, s) : launch_t<1, NT_>(ctx, a, s))
    if (groups <= 1) return LUMEN_MMA(1);
    if (groups <= 2) return LUMEN_MMA(2);
    if (groups <= 4) return LUMEN_MMA(4);
    return LUMEN_MMA(8);
#undef LUMEN_MMA
}

}  // namespace lumen
