// Kernel launchers of the models given as a list of layers (api_decoder.cu): latent attention, grouped-query attention over
// chunks, matrix-memory layers, routed experts, outputs normed before they are added to the residual, bigram and per-layer
// token inputs.  Constants are parameters.
#pragma once

#include "common.cuh"

namespace lumen {

// ---- embedding (decoder_embed.cu) -----------------------------------------------------------------
// x[m] = embed[id] * scale (+ bigram[row]), row = (previous id * mul_prev + id * mul_cur) mod buckets, `buckets` for the first
// token of a sequence.  Row m = b * S + s; the token before s == 0 is last_tok[b], absent when *d_len == 0.
struct EmbedArgs {
    const float *ids = nullptr;  // [B * S]
    const void *embed = nullptr, *bigram = nullptr;
    lumen_dtype dt = LUMEN_F32;
    size_t B = 1, S = 1, vocab = 0, dim = 0, buckets = 0, mul_prev = 0, mul_cur = 0;
    const int *d_len = nullptr, *last_tok = nullptr;
    float scale = 1.f;
    float *x = nullptr;
    // With norm_w the first layer reads RMSNorm(x) * norm_w; what it reads as f32 and/or as a bf16 split (null: not stored)
    const float *norm_w = nullptr;
    float eps = 0.f;
    float *out = nullptr;
    __nv_bfloat16 *hi = nullptr, *lo = nullptr;
};
int launch_embed(lumen_ctx *ctx, const EmbedArgs &a, cudaStream_t s);
// End of a step: every layer's cache grows by S rows and last_tok[b] becomes the id of the sequence's last token.
int launch_advance(lumen_ctx *ctx, int *d_lens, size_t layers, const float *ids, int *last_tok, size_t B, size_t S, cudaStream_t s);

// ---- finishing a product of several rows (gemm_finish.cu) ------------------------------------------
// What follows the sum of a product's split-K slices.  Activations are written as f32 and/or as a bf16 hi/lo pair.
struct StepFinish {
    enum Kind {
        kStore,     // out = sum
        kNormAdd,   // x += RMSNorm(sum + gathered rows) * gain; then of x, or of RMSNorm(x) * next_gain: out, (hi, lo) = split
        kGelu,      // out = gelu_tanh(sum)
        kSideGate,  // out = gelu_tanh(sum) * table[id, col]
        kGated,     // sum holds gate and up in blocks of 64 columns: out = glu(gate, up)
    } kind = kStore;
    float *x = nullptr;
    const float *gain = nullptr, *next_gain = nullptr;
    float eps = 0.f;
    const __nv_bfloat16 *gather_src = nullptr;  // rows gather_idx[row, 0 .. gather_n) of this matrix are added too
    const int *gather_idx = nullptr;
    int gather_n = 0;
    const float *ids = nullptr;         // kSideGate
    const void *table = nullptr;
    lumen_dtype table_dt = LUMEN_F32;
    size_t table_ld = 0, table_rows = 0;
    enum Glu { kClampedSwish, kGeluTanh } glu = kClampedSwish;  // kGated: see gated_act / gelu_tanh(gate) * up
    float limit = 0.f;
    size_t ff = 0;
    float *out = nullptr;
    __nv_bfloat16 *hi = nullptr, *lo = nullptr;
};
// part: [splits][rows][n] (null with kNormAdd: nothing but gathered rows).
int launch_step_finish(lumen_ctx *ctx, const float *part, int splits, size_t rows, size_t n, const StepFinish &f, cudaStream_t s);

// ---- products -----------------------------------------------------------------------------------
// C = A . W^T with bf16 operands on the tensor cores: A as one bf16 matrix (a_lo null) or as a hi/lo pair.
struct GemmBf16Args {
    const __nv_bfloat16 *a_hi = nullptr, *a_lo = nullptr;
    size_t M = 0, K = 0, lda = 0;  // lda, ldw in elements (0: K)
    const __nv_bfloat16 *w = nullptr;
    size_t N = 0, ldw = 0;
    float *c = nullptr;                // [M, N] f32 (scratch when a finisher follows)
    const StepFinish *fin = nullptr;
    __nv_bfloat16 *out16 = nullptr;    // instead of c: bf16 result of the epilogue
    size_t ld16 = 0;
    enum Epi { kF32 = 0, kBf16 = 1, kGelu = 2, kGated = 3, kGatedGelu = 4 } epi = kF32;
    float limit = 0.f;                 // kGated, kGatedGelu: N = 2 * 64 * ceil(ff / 64) interleaved rows, ff columns stored
    size_t ff = 0;
    // Grouped: tile t covers rows tiles[t].x .. tiles[t].y - 1 of A against the N rows of W from tiles[t].z * N;
    // tiles beyond *n_tiles are empty.  row_scale multiplies a row's sums before the activation.
    const int4 *tiles = nullptr;
    const int *n_tiles = nullptr;
    size_t max_tiles = 0, w_groups = 1;
    const float *row_scale = nullptr;
};
bool gemm_bf16_usable(size_t K, size_t lda, size_t ldw, const void *a, const void *w);
int launch_gemm_bf16(lumen_ctx *ctx, const GemmBf16Args &g, cudaStream_t s);
// C[M,N] = A . W^T in 32-bit FMAs, whatever the sizes.
int launch_gemm_simt(lumen_ctx *ctx, const float *a, const void *w, lumen_dtype wdt, float *c, size_t M, size_t K, size_t N,
                     const float *residual, cudaStream_t s);

// One row.  The vector arrives as `res`, optionally with a sublayer's output still to be normed and added:
// x = res + RMSNorm(y) * gain, stored to x_out by the first CTA (x_out != res); then optionally RMSNorm(x) * norm_w.
struct GemvStepArgs {
    const float *res = nullptr, *y = nullptr, *gain = nullptr;
    float *x_out = nullptr;
    const float *norm_w = nullptr;
    float eps = 0.f;
    const void *w = nullptr;
    lumen_dtype wdt = LUMEN_F32;
    size_t K = 0, N = 0;
    float *out = nullptr;
    StepFinish::Kind act = StepFinish::kStore;  // kStore, kGelu, kSideGate, or kGated (gelu_tanh(gate) * up; N = ff)
    const float *ids = nullptr;
    const void *table = nullptr;
    size_t table_ld = 0, table_rows = 0;
};
int launch_gemv_step(lumen_ctx *ctx, const GemvStepArgs &a, cudaStream_t s);

// ---- routed experts (moe.cu) -----------------------------------------------------------------------
// Gate and up rows of one feed-forward are stored in blocks: 64 gate rows, then the 64 up rows that go with them.
constexpr size_t kGateBlock = 64;
inline size_t gated_rows(size_t ff) { return (ff + kGateBlock - 1) / kGateBlock * 2 * kGateBlock; }
struct MoeArgs {
    size_t M = 0, W = 0, experts = 0, top = 0, ff = 0, shared_ff = 0;
    float limit = 0.f, shared_limit = 0.f;
    lumen_dtype wdt = LUMEN_F32;
    const float *x = nullptr, *z = nullptr;  // [M, W], router logits [M, experts]
    const void *gate_up = nullptr, *down = nullptr, *shared_gate_up = nullptr, *shared_down = nullptr;
    float *act = nullptr;  // [M, top * ff + shared_ff]
    int *sel = nullptr;    // [M, top] chosen experts
    float *y = nullptr;    // [M, W]
};
bool moe_vec_usable(const MoeArgs &a);
int launch_moe_vec(lumen_ctx *ctx, const MoeArgs &a, cudaStream_t s);
// Many rows: choose, group the rows by expert, gather them.
struct MoeGroupArgs {
    size_t M = 0, experts = 0, top = 0;
    const float *z = nullptr;
    int *sel = nullptr, *pos = nullptr, *src = nullptr;  // [M, top], [M, top], [M * top]
    float *weight = nullptr, *row_scale = nullptr;       // [M, top], [M * top]
    int4 *tiles = nullptr;
    int *n_tiles = nullptr;
};
inline size_t moe_max_tiles(size_t M, size_t experts, size_t top) { return M * top / 128 + (experts < M * top ? experts : M * top); }
int launch_moe_group(lumen_ctx *ctx, const MoeGroupArgs &a, cudaStream_t s);
int launch_gather_rows(lumen_ctx *ctx, const __nv_bfloat16 *in, const int *src, __nv_bfloat16 *out, size_t rows, size_t dim, cudaStream_t s);

// ---- latent attention (latent_attention.cu, latent_attn_mma.cu, attn_prefill_tc.cu) ----------------
// u[M, u_ld] holds per row the queries (head by head: dim unrotated, rot_dim rotated numbers), the latent and the shared
// key part (kv_rank + rot_dim numbers) at u_kv, and the heads' gate logits at u_gate.  Cache row: latent, rotated key part,
// zeros up to `pitch`.  T = element type of the cache, of qf and of the expanded operands: f32, or bf16 in bf16 models.
struct LatentArgs {
    size_t B = 0, S = 0, H = 0, dim = 0, rot_dim = 0, vdim = 0, rank = 0, rot_dims = 0, pitch = 0, max_seq = 0;
    lumen_dtype dt = LUMEN_F32;
    const float *u = nullptr;
    size_t u_ld = 0, u_kv = 0, u_gate = 0;
    const float *latent_gain = nullptr;
    float eps = 0.f, scale = 0.f;
    const float *cos_t = nullptr, *sin_t = nullptr;  // [max_seq, rot_dims / 2]
    const void *wuk = nullptr, *wuv = nullptr;
    void *cache = nullptr;                           // [B, max_seq, pitch]
    const int *d_len = nullptr;                      // rows cached before this step
    size_t past = 0;                                 // the host's view of *d_len
    void *qf = nullptr;                              // [B * S * H, pitch]: W_uk^T q per head, rotated part, zeros
    float *part_ctx = nullptr, *part_ml = nullptr;   // [rows, nsplit, rank], [rows, nsplit, 2]
    int nsplit = 1;
    float *out = nullptr;                            // [M, H * vdim] (null: not stored)
    __nv_bfloat16 *out_hi = nullptr, *out_lo = nullptr;
};
// Latent normed, key part rotated, both appended to the cache.
int launch_latent_append(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s);
// qf, and (append) the cache rows in the same launch.
int launch_latent_absorb(lumen_ctx *ctx, const LatentArgs &a, bool append, cudaStream_t s);
// Scores and weighted latents of every query row over the cached rows, in nsplit pieces.
int latent_pick_splits(const LatentArgs &a, size_t total, int num_sms);
bool latent_mma_usable(const LatentArgs &a);
int launch_latent_scores(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s);
int launch_latent_mma(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s);
// Cached rows a piece is made of: pieces of one tile each while there are fewer tiles than pieces, else about equal shares.
constexpr int kLatentTile = 64;
#ifdef __CUDACC__
__device__ __forceinline__ int latent_pieces(int total, int nsplit) { return min(nsplit, (total + kLatentTile - 1) / kLatentTile); }
__device__ __forceinline__ int latent_piece_start(int total, int pieces, int i) {  // first cached row of piece i (i == pieces: the end)
    return (int)((long long)i * ((total + kLatentTile - 1) / kLatentTile) / pieces) * kLatentTile;
}
#endif
// Pieces merged, W_uv and the output gate applied.
int launch_latent_value(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s);
// Whole portions on the tensor cores over expanded keys and values (bf16); the cache already holds the rows.
bool latent_prefill_usable(const LatentArgs &a);
int launch_latent_prefill(lumen_ctx *ctx, const LatentArgs &a, cudaStream_t s);

// ---- matrix-memory layers (mlstm.cu, mlstm_chunk_tc.cu) ---------------------------------------------
// Per head: S <- exp(f + m - m') S + exp(i - m') k v^T, n likewise with k alone, m' = max(f + m, i);
// o = S^T q / (max(|n . q|, exp(-m')) + 1e-6), RMS-normed per head, times head_gain and sigmoid(g).
struct MlstmArgs {
    size_t B = 0, S = 0, H = 0, dim = 0, vdim = 0;
    float cap = 0.f, eps = 0.f;
    // Projections of row m: f32 at u + m * u_ld (queries at 0, keys at u_k, values at u_v, output gates at u_g), or bf16 at u16
    // with the same offsets (chunked form).
    const float *u = nullptr;
    const __nv_bfloat16 *u16 = nullptr;
    size_t u_ld = 0, u_k = 0, u_v = 0, u_g = 0;
    const float *z = nullptr, *z_bias = nullptr;  // gate pre-activations z[m * z_ld + h] (input) and [.. + H + h] (forget), biases [2 H]
    size_t z_ld = 0;
    const float *head_gain = nullptr;             // [H * vdim]
    float *state = nullptr, *norm = nullptr, *mx = nullptr;  // [B, H, dim, vdim], [B, H, dim], [B, H]; absent while *d_len == 0
    const int *d_len = nullptr;
    size_t past = 0;                              // the host's view of *d_len
    float *out = nullptr;                         // [B * S, H * vdim] (null: not stored)
    __nv_bfloat16 *out_hi = nullptr, *out_lo = nullptr;
};
// Token by token, any sizes.
int launch_mlstm_step(lumen_ctx *ctx, const MlstmArgs &a, cudaStream_t s);
// Portions in chunks of kMlstmChunk tokens on the tensor cores (bf16 projections).
constexpr int kMlstmChunk = 128;
bool mlstm_chunked_usable(const MlstmArgs &a);
int launch_mlstm_chunked(lumen_ctx *ctx, const MlstmArgs &a, cudaStream_t s);

// ---- grouped-query attention over chunks (grouped_attention.cu, attn_prefill_tc.cu) ----------------
// u[M, u_ld] holds per row the queries (H x dim), and for layers with keys and values of their own the keys (G x dim) at u_k
// and values (G x vdim) at u_v, and the heads' gate logits at u_gate.  T = element type of the cache: f32, or bf16 in bf16 models.
struct GroupedArgs {
    size_t B = 0, S = 0, H = 0, G = 0, dim = 0, vdim = 0, rot_dims = 0, chunk = 0, max_seq = 0;
    lumen_dtype dt = LUMEN_F32;
    const float *u = nullptr;
    size_t u_ld = 0, u_k = 0, u_v = 0, u_gate = 0;
    bool own_kv = true;
    const float *q_gain = nullptr, *k_gain = nullptr, *sink = nullptr;  // [dim], [dim], [H]
    float eps = 0.f, scale = 0.f;
    const float *cos_t = nullptr, *sin_t = nullptr;                     // [max_seq, rot_dims / 2]
    void *k = nullptr, *v = nullptr;                                    // [B, G, max_seq, dim], [B, G, max_seq, vdim]
    const int *d_len = nullptr;
    size_t past = 0;
    float *part_ctx = nullptr, *part_ml = nullptr;  // [rows * H, nsplit, vdim], [rows * H, nsplit, 2]
    int nsplit = 1;
    float *out = nullptr;                           // [M, H * vdim] (null: not stored)
    __nv_bfloat16 *out_hi = nullptr, *out_lo = nullptr;
};
constexpr size_t kGroupedMaxDim = 512;
int grouped_pick_splits(const GroupedArgs &a, int num_sms);
// Keys (normed, rotated) and values -> cache, for layers with keys and values of their own; with q also the queries
// (normed, rotated) as bf16 [B, H, s_pad, width].
int launch_grouped_append(lumen_ctx *ctx, const GroupedArgs &a, __nv_bfloat16 *q, size_t s_pad, size_t width, cudaStream_t s);
// Attention of every row over the cached rows in nsplit pieces, merged with the sink and the gate.  append: the one new row of
// every sequence (S == 1) is appended by the same launch.
int launch_grouped_attention(lumen_ctx *ctx, const GroupedArgs &a, bool append, cudaStream_t s);
// Whole portions on the tensor cores (bf16), append included.
bool grouped_prefill_usable(const GroupedArgs &a);
int launch_grouped_prefill(lumen_ctx *ctx, const GroupedArgs &a, cudaStream_t s);
// out[(b * heads + h) * cols + c][j] = in[b][h][row0 + j][c], j < rows (zeros up to the pitch): rows of a cache as columns.
int launch_transpose_rows(lumen_ctx *ctx, const __nv_bfloat16 *in, size_t in_rows, size_t cols, size_t mats, size_t row0, size_t rows,
                          __nv_bfloat16 *out, size_t pitch, cudaStream_t s);

// ---- shared device helpers ----------------------------------------------------------------------
#ifdef __CUDACC__
// 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3)))
__device__ __forceinline__ float gelu_tanh(float z) {
    const float t = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
    return 0.5f * z * (1.0f + tanhf(t));
}
__device__ __forceinline__ float sigmoid_f(float z) { return __fdiv_rn(1.0f, 1.0f + expf(-z)); }
// min(g, limit) * sigmoid(1.702 min(g, limit)) * (clamp(u, -limit, limit) + 1)
__device__ __forceinline__ float gated_act(float g, float u, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoid_f(1.702f * g) * (u + 1.0f);
}
__device__ __forceinline__ unsigned long long id_to_index(float f) {  // `as usize` saturates; NaN and negatives become 0
    return (f != f || f <= 0.f) ? 0ull : (f >= 1.8e19f ? ~0ull : (unsigned long long)f);
}
template <typename T>
__device__ __forceinline__ float to_f32(T v) {
    if constexpr (sizeof(T) == 4) return v;
    else return __bfloat162float(v);
}
template <typename T>
__device__ __forceinline__ T from_f32(float v) {
    if constexpr (sizeof(T) == 4) return v;
    else return __float2bfloat16_rn(v);
}
__device__ __forceinline__ float table_at(const void *t, lumen_dtype dt, size_t i) {
    return dt == LUMEN_F32 ? static_cast<const float *>(t)[i] : __bfloat162float(static_cast<const __nv_bfloat16 *>(t)[i]);
}
__device__ __forceinline__ void store_split(float v, __nv_bfloat16 *hi, __nv_bfloat16 *lo, size_t i) {
    const __nv_bfloat16 h = __float2bfloat16_rn(v);
    hi[i] = h;
    if (lo) lo[i] = __float2bfloat16_rn(v - __bfloat162float(h));
}
#endif

}  // namespace lumen
