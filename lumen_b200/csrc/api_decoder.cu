// C ABI: models given as a list of layers (lumen_decoder_new) on one GPU; the entry points they share with LlamaModel are in
// model_base.cu.
//
// Memory: one device slab holds every weight (the projections that read a layer's input are stored back to back, so that they are
// one product; gate and up rows of a gated feed-forward alternate in blocks of 64, experts follow one another), one slab per set
// of caches holds what all layers keep (latents, keys and values, or a recurrent state), one workspace the activations.  A
// sequence's state is its layers' caches and its last token id (the bigram embedding looks back across steps); a recurrent
// state counts as zeros while the sequence has no positions, so that resetting a cache resets its length alone.
//
// A step of one row streams the weights through vector-matrix kernels; the norm of a sublayer's output, the residual sum
// and the norm before the next sublayer are formed by the kernel that reads the result next.  It is captured once per split count into a CUDA graph.  Steps of
// several rows run every product on the tensor cores (bf16 models) with finishing kernels that write the next product's operand.
#include <algorithm>
#include <cmath>

#include "decoder_kernels.cuh"
#include "model_base.cuh"

using namespace lumen;

namespace {

struct Slot {  // where a parameter goes
    char *dst = nullptr;
    size_t rows = 0, cols = 0;  // cols == 0: vector of `rows`
    lumen_dtype dt = LUMEN_F32;
    bool plus_one = false;      // gains stored around zero: 1 + w is kept
    int half = -1;              // 0 / 1: gate / up rows of a gated feed-forward (blocks of kGateBlock)
};

struct LayerW {
    // [proj_rows, W].  Latent attention: queries, latent and shared key part (u_kv), gates (u_gate).  Attention: queries, keys (u_k)
    // and values (u_v) where the layer has its own, gates (u_gate).  Matrix memory: queries, keys (u_k), values (u_v), output
    // gates (u_gate), and the 2 H rows of the input and forget gates, which are a product of their own in steps of several rows.
    char *proj = nullptr;
    char *uk = nullptr, *uv = nullptr, *o = nullptr;
    float *latent_gain = nullptr, *side_norm = nullptr;
    float *pre1 = nullptr, *pre2 = nullptr;                   // gains of the norms before the sublayers (null: none)
    float *norm1 = nullptr, *norm2 = nullptr;                 // gains of the norms of their outputs
    float *q_gain = nullptr, *k_gain = nullptr, *sink = nullptr;  // attention
    float *z_bias = nullptr, *head_gain = nullptr;            // matrix memory
    char *up = nullptr, *down = nullptr;                      // dense (up: gate and up rows where it is gated)
    char *router = nullptr, *gate_up = nullptr, *edown = nullptr;  // experts
    char *sgate_up = nullptr, *sdown = nullptr;               // shared expert
    char *side_gate = nullptr, *side_proj = nullptr;
    float *cos_t = nullptr, *sin_t = nullptr;
    size_t proj_rows = 0, main_rows = 0, u_kv = 0, u_k = 0, u_v = 0, u_gate = 0, pitch = 0;  // main_rows: without the 2 H gate rows
};

// An activation matrix as the next product reads it: f32, or bf16 hi (and lo).
struct Act {
    float *f = nullptr;
    __nv_bfloat16 *hi = nullptr, *lo = nullptr;
};

struct Workspace {
    size_t M = 0;
    char *base = nullptr;
    float *x[2] = {nullptr, nullptr}, *u = nullptr, *y = nullptr, *c = nullptr, *nx = nullptr, *last_x = nullptr;
    Act xa, att, act, side;  // xa: what the next sublayer reads (xa.f is the residual itself in models without norms before them)
    void *qf = nullptr;
    float *part_ctx = nullptr, *part_ml = nullptr;
    // experts
    float *z = nullptr, *weight = nullptr, *row_scale = nullptr, *vec_act = nullptr;
    int *sel = nullptr, *pos = nullptr, *src = nullptr, *n_tiles = nullptr;
    int4 *tiles = nullptr;
    __nv_bfloat16 *xperm = nullptr, *aperm = nullptr, *yexp = nullptr;
    float *ids = nullptr, *logits = nullptr, *h_ids = nullptr, *h_logits = nullptr;
    size_t h_logits_elems = 0;
};

// A sublayer's output that is still to be normed and added to the residual.
struct Pending {
    const float *y = nullptr, *gain = nullptr;
};

struct lumen_decoder : lumen_model {
    lumen_decoder_config cfg{};
    std::vector<lumen_decoder_layer> lc;
    std::vector<LayerW> lw;
    size_t W = 0, esz = 4, stream_bytes = 0;
    lumen_dtype dt = LUMEN_F32;
    char *wslab = nullptr;
    char *embed = nullptr, *bigram = nullptr, *side_embed = nullptr, *head = nullptr;
    float *final_gain = nullptr;
    std::map<std::string, Slot> slots;
    Workspace ws;

    ~lumen_decoder() override;
    int build();
    int set_param(const char *name, const void *host_data, const size_t *shape, int ndim, lumen_dtype dtype) override;
    int init_kv_caches(size_t batch, lumen_kv_cache **out) override;
    int check_caches(size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches) override;
    int ensure_workspace(size_t rows) override;
    int run_forward(size_t b, size_t s, lumen_kv_cache **caches, bool last_only) override;
    size_t weight_bytes() const override { return stream_bytes; }

    void cache_shape(size_t l, lumen_kv_cache *c) const;
    int rotation_tables(size_t l, float *cos_t, float *sin_t);
    bool norms_before() const { return cfg.norms == LUMEN_NORM_BOTH; }
    LatentArgs latent_args(size_t l, lumen_kv_cache *c, size_t B, size_t S) const;
    GroupedArgs grouped_args(size_t l, lumen_kv_cache *c, size_t B, size_t S) const;
    MlstmArgs mlstm_args(size_t l, lumen_kv_cache *c, size_t B, size_t S) const;
    int pick_splits(size_t l, lumen_kv_cache *c, size_t B, size_t S) const;  // pieces of the context in the row kernels (1: no such thing)
    int mix_rows(size_t l, lumen_kv_cache *c, size_t B, size_t S);           // projections and mixer of a step of several rows -> ws.att
    MoeArgs moe_args(size_t l, size_t M) const;
    int step_row(lumen_kv_cache **caches);
    int step_rows(size_t B, size_t S, lumen_kv_cache **caches, bool last_only);
    int product(const Act &a, size_t lda, const void *w, size_t M, size_t K, size_t N, float *c, const StepFinish *fin, bool pair = false);
    bool on_tensor_cores(size_t M, size_t K) const;
};

lumen_decoder::~lumen_decoder() {
    if (ws.base) cudaFree(ws.base);
    if (ws.h_ids) cudaFreeHost(ws.h_ids);
    if (ws.h_logits) cudaFreeHost(ws.h_logits);
    if (wslab) cudaFree(wslab);
}

int lumen_decoder::build() {
    const bool bigram_on = cfg.bigram_buckets > 0, side_on = cfg.side_dim > 0;
    size_t off = 0;
    auto take = [&](size_t bytes) { size_t o = off; off += align_up(bytes, 256); return o; };
    // Offsets first (dst holds the offset until the slab exists).
    auto add = [&](const std::string &name, size_t at, size_t rows, size_t cols, lumen_dtype d, bool plus_one = false, int half = -1) {
        Slot s;
        s.dst = reinterpret_cast<char *>(at);
        s.rows = rows; s.cols = cols; s.dt = d; s.plus_one = plus_one; s.half = half;
        slots[name] = s;
    };
    auto matrix = [&](const std::string &name, size_t rows, size_t cols) {
        const size_t o = take(rows * cols * esz);
        add(name, o, rows, cols, dt);
        return o;
    };
    auto vec = [&](const std::string &name, size_t n, bool plus_one) {
        const size_t o = take(n * 4);
        add(name, o, n, 0, LUMEN_F32, plus_one);
        return o;
    };
    struct Off {
        size_t proj, uk = 0, uv = 0, o, lg = 0, n1, n2 = 0, p1 = 0, p2 = 0, qg = 0, kg = 0, sink = 0, zb = 0, hg = 0, sn = 0, up = 0, down = 0, router = 0,
            gu = 0, ed = 0, sgu = 0, sd = 0, sg = 0, sp = 0, cos, sin;
    };
    std::vector<Off> lo(L);
    const size_t o_embed = matrix("embed", V, W);
    const size_t o_bigram = bigram_on ? matrix("bigram", cfg.bigram_buckets + 1, W) : 0;
    const size_t o_side = side_on ? matrix("side.embed", V, L * cfg.side_dim) : 0;
    stream_bytes = 0;
    for (size_t l = 0; l < L; ++l) {
        const lumen_decoder_layer &c = lc[l];
        LayerW &w = lw[l];
        Off &f = lo[l];
        const std::string p = "l" + std::to_string(l) + ".";
        // projections of the layer's input, back to back: (name, rows)
        struct Part { const char *name = ""; size_t rows = 0; };
        Part parts[6];
        const size_t H = c.heads;
        if (c.mixer == LUMEN_MIXER_LATENT) {
            const size_t qn = H * (c.dim + c.rot_dim), kvn = c.kv_rank + c.rot_dim;
            parts[0] = {"q", qn}; parts[1] = {"dkv", kvn}; parts[2] = {"g", H};
            w.u_kv = qn; w.u_gate = qn + kvn;
            w.pitch = align_up(kvn, 16);
        } else if (c.mixer == LUMEN_MIXER_ATTENTION) {
            const size_t kn = c.kv_from < 0 ? c.kv_heads * c.dim : 0, vn = c.kv_from < 0 ? c.kv_heads * c.vdim : 0;
            parts[0] = {"q", H * c.dim}; parts[1] = {"k", kn}; parts[2] = {"v", vn}; parts[3] = {"g", H};
            w.u_k = H * c.dim; w.u_v = w.u_k + kn; w.u_gate = w.u_v + vn;
        } else {
            parts[0] = {"q", H * c.dim}; parts[1] = {"k", H * c.dim}; parts[2] = {"v", H * c.vdim}; parts[3] = {"g", H * c.vdim};
            parts[4] = {"i", H}; parts[5] = {"f", H};
            w.u_k = H * c.dim; w.u_v = 2 * H * c.dim; w.u_gate = w.u_v + H * c.vdim;
        }
        for (const Part &q : parts) w.proj_rows += q.rows;
        w.main_rows = w.proj_rows - (c.mixer == LUMEN_MIXER_MLSTM ? 2 * H : 0);
        f.proj = take(w.proj_rows * W * esz);
        size_t at_row = 0;
        for (const Part &q : parts) {
            if (q.rows) add(p + "mix." + q.name, f.proj + at_row * W * esz, q.rows, W, dt);
            at_row += q.rows;
        }
        stream_bytes += w.proj_rows * W * esz;
        if (c.mixer == LUMEN_MIXER_LATENT) {
            f.lg = vec(p + "mix.dkv.norm", c.kv_rank, false);
            f.uk = matrix(p + "mix.uk", H * c.dim, c.kv_rank);
            f.uv = matrix(p + "mix.uv", H * c.vdim, c.kv_rank);
            stream_bytes += H * (c.dim + c.vdim) * c.kv_rank * esz;
        } else if (c.mixer == LUMEN_MIXER_ATTENTION) {
            f.qg = vec(p + "mix.q.norm", c.dim, false);
            if (c.kv_from < 0) f.kg = vec(p + "mix.k.norm", c.dim, false);
            f.sink = vec(p + "mix.sink", H, false);
        } else {
            f.hg = vec(p + "mix.norm", H * c.vdim, false);
            f.zb = take(2 * H * 4);
            add(p + "mix.i.b", f.zb, H, 0, LUMEN_F32);
            add(p + "mix.f.b", f.zb + H * 4, H, 0, LUMEN_F32);
        }
        f.o = matrix(p + "mix.o", W, H * c.vdim);
        stream_bytes += W * H * c.vdim * esz;
        const bool both = norms_before();  // norm<i> before and norm<i>b after a sublayer, gains as they are; else norm<i> after it, around one
        if (both) f.p1 = vec(p + "norm1", W, false);
        f.n1 = vec(p + (both ? "norm1b" : "norm1"), W, !both);
        auto gated = [&](const std::string &name, size_t at, size_t ff) {
            add(name + ".gate", at, ff, W, dt, false, 0);
            add(name + ".up", at, ff, W, dt, false, 1);
        };
        if (c.mlp_kind != LUMEN_MLP_NONE) {
            if (both) f.p2 = vec(p + "norm2", W, false);
            f.n2 = vec(p + (both ? "norm2b" : "norm2"), W, !both);
        }
        if (c.mlp_kind == LUMEN_MLP_DENSE) {
            f.up = matrix(p + "mlp.up", c.ff, W);
            f.down = matrix(p + "mlp.down", W, c.ff);
            stream_bytes += 2 * c.ff * W * esz;
        } else if (c.mlp_kind == LUMEN_MLP_GATED_GELU) {
            f.up = take(gated_rows(c.ff) * W * esz);
            gated(p + "mlp", f.up, c.ff);
            f.down = matrix(p + "mlp.down", W, c.ff);
            stream_bytes += 3 * c.ff * W * esz;
        } else if (c.mlp_kind == LUMEN_MLP_MOE) {
            const size_t gr = gated_rows(c.expert_ff);
            f.router = matrix(p + "mlp.router", c.experts, W);
            f.gu = take(c.experts * gr * W * esz);
            f.ed = take(c.experts * W * c.expert_ff * esz);
            for (size_t e = 0; e < c.experts; ++e) {
                const std::string n = p + "mlp.e" + std::to_string(e);
                gated(n, f.gu + e * gr * W * esz, c.expert_ff);
                add(n + ".down", f.ed + e * W * c.expert_ff * esz, W, c.expert_ff, dt);
            }
            if (c.shared_ff) {
                f.sgu = take(gated_rows(c.shared_ff) * W * esz);
                gated(p + "mlp.shared", f.sgu, c.shared_ff);
                f.sd = matrix(p + "mlp.shared.down", W, c.shared_ff);
            }
            stream_bytes += (c.experts + 3 * (c.top * c.expert_ff + c.shared_ff)) * W * esz;
        }
        if (side_on) {
            f.sg = matrix(p + "side.gate", cfg.side_dim, W);
            f.sp = matrix(p + "side.proj", W, cfg.side_dim);
            f.sn = vec(p + "side.norm", W, false);
            stream_bytes += 2 * cfg.side_dim * W * esz;
        }
        // layers that turn alike share their tables
        f.cos = f.sin = 0;
        for (size_t k = 0; k < l && !f.cos; ++k)
            if (lc[k].rot_dims == c.rot_dims && lc[k].rot_base == c.rot_base && lc[k].rot_factor == c.rot_factor && lc[k].rot_low == c.rot_low &&
                lc[k].rot_high == c.rot_high && lc[k].rot_original == c.rot_original) { f.cos = lo[k].cos; f.sin = lo[k].sin; }
        if (!f.cos) {
            f.cos = take(cfg.max_seq_len * (c.rot_dims / 2) * 4);
            f.sin = take(cfg.max_seq_len * (c.rot_dims / 2) * 4);
        }
    }
    const size_t o_fn = vec("final.norm", W, !norms_before()), o_head = cfg.tied_head ? o_embed : matrix("head", V, W);
    stream_bytes += V * W * esz;
    LUMEN_CUDA(ctx, cudaMalloc(&wslab, std::max<size_t>(off, 256)));
    LUMEN_CUDA(ctx, cudaMemsetAsync(wslab, 0, off, ctx->stream));  // (blocks of gate and up rows are padded with zeros)
    LUMEN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    for (auto &kv : slots) kv.second.dst = wslab + reinterpret_cast<size_t>(kv.second.dst);
    auto at = [&](size_t o) { return wslab + o; };
    auto atf = [&](size_t o) { return reinterpret_cast<float *>(wslab + o); };
    embed = at(o_embed); bigram = bigram_on ? at(o_bigram) : nullptr; side_embed = side_on ? at(o_side) : nullptr;
    final_gain = atf(o_fn); head = at(o_head);
    for (size_t l = 0; l < L; ++l) {
        LayerW &w = lw[l];
        const Off &f = lo[l];
        w.proj = at(f.proj); w.uk = at(f.uk); w.uv = at(f.uv); w.o = at(f.o); w.latent_gain = atf(f.lg); w.norm1 = atf(f.n1);
        if (norms_before()) { w.pre1 = atf(f.p1); w.pre2 = atf(f.p2); }
        w.q_gain = atf(f.qg); w.k_gain = atf(f.kg); w.sink = atf(f.sink); w.z_bias = atf(f.zb); w.head_gain = atf(f.hg);
        w.norm2 = atf(f.n2); w.up = at(f.up); w.down = at(f.down); w.router = at(f.router); w.gate_up = at(f.gu); w.edown = at(f.ed);
        w.sgate_up = at(f.sgu); w.sdown = at(f.sd); w.side_gate = at(f.sg); w.side_proj = at(f.sp); w.side_norm = atf(f.sn);
        w.cos_t = atf(f.cos); w.sin_t = atf(f.sin);
        bool first = true;
        for (size_t k = 0; k < l; ++k) first = first && lo[k].cos != f.cos;
        if (first && lc[l].rot_dims) LUMEN_TRY(rotation_tables(l, w.cos_t, w.sin_t));
    }
    n_expected = slots.size();
    return LUMEN_OK;
}

// cos and sin of position * frequency, computed in double.  With frequency scaling, wavelengths above rot_original / rot_low are
// stretched by rot_factor, those below rot_original / rot_high stay, and frequencies between are interpolated.
int lumen_decoder::rotation_tables(size_t l, float *cos_t, float *sin_t) {
    const lumen_decoder_layer &c = lc[l];
    const size_t half = c.rot_dims / 2;
    std::vector<float> ch(cfg.max_seq_len * half), sh(ch.size());
    for (size_t i = 0; i < half; ++i) {
        double freq = std::pow(c.rot_base, -2.0 * (double)i / (double)c.rot_dims);
        if (c.rot_factor != 0.0) {
            const double turns = c.rot_original * freq / (2.0 * M_PI);  // within the original length
            if (turns < c.rot_low) {
                freq /= c.rot_factor;
            } else if (turns <= c.rot_high) {
                const double s = (turns - c.rot_low) / (c.rot_high - c.rot_low);
                freq = (1.0 - s) * freq / c.rot_factor + s * freq;
            }
        }
        for (size_t p = 0; p < cfg.max_seq_len; ++p) {
            ch[p * half + i] = (float)std::cos((double)p * freq);
            sh[p * half + i] = (float)std::sin((double)p * freq);
        }
    }
    LUMEN_CUDA(ctx, cudaMemcpy(cos_t, ch.data(), ch.size() * 4, cudaMemcpyHostToDevice));
    LUMEN_CUDA(ctx, cudaMemcpy(sin_t, sh.data(), sh.size() * 4, cudaMemcpyHostToDevice));
    return LUMEN_OK;
}

int lumen_decoder::set_param(const char *name, const void *host_data, const size_t *shape, int ndim, lumen_dtype dtype) {
    auto it = slots.find(name);
    if (it == slots.end()) return set_error(ctx, LUMEN_ERR_PARAM_NAME, "unknown parameter '%s'", name);
    const Slot &s = it->second;
    if (s.cols == 0) {
        if (ndim != 1 || shape[0] != s.rows) return set_error(ctx, LUMEN_ERR_SHAPE, "%s: expected [%zu]", name, s.rows);
        std::vector<float> v(s.rows);
        for (size_t i = 0; i < s.rows; ++i) {
            float x;
            if (dtype == LUMEN_F32) {
                x = static_cast<const float *>(host_data)[i];
            } else {
                const uint32_t bits = (uint32_t)static_cast<const uint16_t *>(host_data)[i] << 16;
                memcpy(&x, &bits, 4);
            }
            v[i] = s.plus_one ? 1.0f + x : x;
        }
        LUMEN_TRY(upload_block(ctx, s.dst, LUMEN_F32, v.data(), LUMEN_F32, 1, s.rows, 0, s.rows));
    } else {
        if (ndim != 2 || shape[0] != s.rows || shape[1] != s.cols)
            return set_error(ctx, LUMEN_ERR_SHAPE, "%s: expected [%zu,%zu]", name, s.rows, s.cols);
        const size_t se = dtype == LUMEN_F32 ? 4 : 2, de = s.dt == LUMEN_F32 ? 4 : 2;
        const size_t block = s.half < 0 ? s.rows : kGateBlock;
        for (size_t r = 0; r < s.rows; r += block) {
            const size_t nr = std::min(block, s.rows - r), dst_row = s.half < 0 ? r : 2 * r + s.half * kGateBlock;
            LUMEN_TRY(upload_block(ctx, s.dst + dst_row * s.cols * de, s.dt, static_cast<const char *>(host_data) + r * s.cols * se, dtype, nr,
                                   s.cols, 0, s.cols));
        }
    }
    is_set[name] = true;
    return LUMEN_OK;
}

// What layer l's cache holds (see lumen_kv_cache).
void lumen_decoder::cache_shape(size_t l, lumen_kv_cache *c) const {
    const lumen_decoder_layer &k = lc[l];
    c->dtype = dt;
    if (k.mixer == LUMEN_MIXER_LATENT) {
        c->kind = lumen_kv_cache::kLatent;
        c->h_kv = 1; c->d = lw[l].pitch;
    } else if (k.mixer == LUMEN_MIXER_ATTENTION) {
        c->kind = lumen_kv_cache::kRows;
        c->h_kv = k.kv_heads; c->d = k.dim; c->dv = k.vdim;
    } else {
        c->kind = lumen_kv_cache::kState;
        c->h_kv = k.heads; c->d = k.dim; c->dv = k.vdim;
        c->dtype = LUMEN_F32;
    }
}

int lumen_decoder::init_kv_caches(size_t batch, lumen_kv_cache **out) {
    if (batch == 0) return set_error(ctx, LUMEN_ERR_SHAPE, "caches for an empty batch");
    std::vector<size_t> at(L), at2(L);
    size_t off = 0;
    auto take = [&](size_t bytes) { const size_t o = off; off += align_up(bytes, 256); return o; };
    for (size_t l = 0; l < L; ++l) {
        const lumen_decoder_layer &k = lc[l];
        if (k.mixer == LUMEN_MIXER_LATENT) {
            at[l] = at2[l] = take(batch * cfg.max_seq_len * lw[l].pitch * esz);
        } else if (k.mixer == LUMEN_MIXER_MLSTM) {
            at[l] = take(batch * k.heads * k.dim * k.vdim * 4);
            at2[l] = take(batch * k.heads * (k.dim + 1) * 4);
        } else if (k.kv_from >= 0) {  // that layer's rows
            at[l] = at[k.kv_from];
            at2[l] = at2[k.kv_from];
        } else {
            at[l] = take(batch * k.kv_heads * cfg.max_seq_len * k.dim * esz);
            at2[l] = take(batch * k.kv_heads * cfg.max_seq_len * k.vdim * esz);
        }
    }
    const size_t lens_at = off, last_at = lens_at + align_up(L * sizeof(int), 256);
    int rc = LUMEN_OK;
    lumen_storage *slab = new_cache_slab(ctx, last_at + align_up(batch * sizeof(int), 256), &rc);
    if (!slab) return rc;
    char *base = static_cast<char *>(slab->ptr);
    for (size_t l = 0; l < L; ++l) {
        auto *c = new lumen_kv_cache();
        const lumen_decoder_layer &k = lc[l];
        c->ctx = ctx; c->b = batch; c->max_seq = cfg.max_seq_len;
        cache_shape(l, c);
        c->k = reinterpret_cast<float *>(base + at[l]);
        if (k.mixer != LUMEN_MIXER_LATENT) c->v = reinterpret_cast<float *>(base + at2[l]);
        c->d_len = reinterpret_cast<int *>(base + lens_at) + l;
        c->last_tok = reinterpret_cast<int *>(base + last_at);
        c->seen_abort = ctx->abort_gen;
        c->owns_slab = false;
        c->slab = slab;
        slab->refs += 1;
        out[l] = c;
    }
    return LUMEN_OK;
}

int lumen_decoder::check_caches(size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches) {
    if (n_caches != L || !caches) return set_error(ctx, LUMEN_ERR_CACHE_COUNT, "KV cache count mismatch: got %zu, expected %zu", n_caches, L);
    for (size_t l = 0; l < L; ++l) {
        lumen_kv_cache *c = caches[l];
        if (!c) return set_error(ctx, LUMEN_ERR_INVALID, "null KV cache for layer %zu", l);
        LUMEN_TRY(kv_resync_len(c));
        lumen_kv_cache want;
        cache_shape(l, &want);
        if (c->b != b || c->kind != want.kind || c->h_kv != want.h_kv || c->d != want.d || c->dv != want.dv || c->dtype != want.dtype ||
            c->max_seq != cfg.max_seq_len || !c->last_tok)
            return set_error(ctx, LUMEN_ERR_SHAPE, "KV cache %zu [%zu,%zu,%zu,%zu] does not match batch %zu / model", l, c->b, c->h_kv, c->max_seq, c->d, b);
        if (c->slab != caches[0]->slab || c->d_len != caches[0]->d_len + l)
            return set_error(ctx, LUMEN_ERR_INVALID, "KV caches come from different sets, or are not in layer order");
        if (c->len != caches[0]->len) return set_error(ctx, LUMEN_ERR_INVALID, "KV caches have different lengths");
        if (c->len + s > c->max_seq) return set_error(ctx, LUMEN_ERR_KV_OVERFLOW, "KV cache overflow: new_len=%zu > max_seq=%zu", c->len + s, c->max_seq);
    }
    return LUMEN_OK;
}

// Products of several rows: bf16 models on the tensor cores when the row length allows TMA.
bool lumen_decoder::on_tensor_cores(size_t M, size_t K) const { return dt == LUMEN_BF16 && M > 1 && gemm_bf16_usable(K, K, K, wslab, wslab); }

int lumen_decoder::ensure_workspace(size_t M) {
    if (M <= ws.M) return LUMEN_OK;
    LUMEN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    drop_graphs();
    if (ws.base) cudaFree(ws.base);
    if (ws.h_ids) cudaFreeHost(ws.h_ids);
    if (ws.h_logits) cudaFreeHost(ws.h_logits);
    ws = Workspace();
    size_t u = 0, att = 0, act = 1, q = 0, ctx_rows = 0, zmax = 0, topmax = 0, permx = 0, perma = 0, vact = 1, tiles = 0, c = W, heads = 0, rank = 0;
    for (size_t l = 0; l < L; ++l) {
        const lumen_decoder_layer &k = lc[l];
        u = std::max(u, lw[l].proj_rows);
        att = std::max(att, k.heads * k.vdim);
        if (k.mixer == LUMEN_MIXER_MLSTM) {
            zmax = std::max(zmax, 2 * k.heads);
        } else {
            q = std::max(q, k.heads * lw[l].pitch);
            heads = std::max(heads, k.heads);
            rank = std::max(rank, k.mixer == LUMEN_MIXER_LATENT ? k.kv_rank : k.vdim);
        }
        if (k.mlp_kind == LUMEN_MLP_DENSE) {
            act = std::max(act, k.ff);
            c = std::max(c, k.ff);
        } else if (k.mlp_kind == LUMEN_MLP_GATED_GELU) {
            act = std::max(act, k.ff);
            c = std::max(c, gated_rows(k.ff));
        } else if (k.mlp_kind == LUMEN_MLP_MOE) {
            act = std::max(act, k.shared_ff);
            c = std::max(c, gated_rows(k.shared_ff));
            zmax = std::max(zmax, k.experts);
            topmax = std::max(topmax, k.top);
            permx = std::max(permx, k.top * W);
            perma = std::max(perma, k.top * k.expert_ff);
            vact = std::max(vact, k.top * k.expert_ff + k.shared_ff);
            tiles = std::max(tiles, moe_max_tiles(M, k.experts, k.top));
        }
    }
    ctx_rows = std::max(M * heads, (size_t)ctx->num_sms * 2 * 32);
    const bool bf = dt == LUMEN_BF16;
    size_t off = 0;
    auto take = [&](size_t bytes) { size_t o = off; off += align_up(bytes, 256); return o; };
    const size_t sd = cfg.side_dim;
    const size_t o_x0 = take(M * W * 4), o_x1 = take(M * W * 4), o_u = take(M * u * 4), o_y = take(M * W * 4), o_c = take(M * std::max(c, sd) * 4),
                 o_nx = take(M * W * 4), o_last = take(M * W * 4), o_att = take(M * att * 4), o_act = take(M * act * 4), o_sd = take(M * sd * 4),
                 o_xh = take(bf ? M * W * 2 : 0), o_xl = take(bf ? M * W * 2 : 0), o_ah = take(bf ? M * att * 2 : 0), o_gh = take(bf ? M * act * 2 : 0),
                 o_sh = take(bf ? M * sd * 2 : 0), o_q = take(M * q * esz), o_pc = take(ctx_rows * rank * 4), o_pm = take(ctx_rows * 8),
                 o_z = take(M * zmax * 4), o_wt = take(M * topmax * 4), o_rs = take(M * topmax * 4), o_ye = take(bf ? M * topmax * W * 2 : 0),
                 o_va = take(M * vact * 4), o_sel = take(M * topmax * 4), o_pos = take(M * topmax * 4), o_src = take(M * topmax * 4), o_nt = take(4),
                 o_tiles = take(tiles * sizeof(int4)), o_xp = take(bf ? M * permx * 2 : 0), o_ap = take(bf ? M * perma * 2 : 0),
                 o_ids = take(M * 4), o_lg = take(M * V * 4), o_xn = take(norms_before() ? M * W * 4 : 0);
    LUMEN_CUDA(ctx, cudaMalloc(&ws.base, off));
    auto f = [&](size_t o) { return reinterpret_cast<float *>(ws.base + o); };
    auto h = [&](size_t o) { return reinterpret_cast<__nv_bfloat16 *>(ws.base + o); };
    auto i = [&](size_t o) { return reinterpret_cast<int *>(ws.base + o); };
    ws.x[0] = f(o_x0); ws.x[1] = f(o_x1); ws.u = f(o_u); ws.y = f(o_y); ws.c = f(o_c); ws.nx = f(o_nx); ws.last_x = f(o_last);
    ws.xa.f = norms_before() ? f(o_xn) : ws.x[0];
    ws.att.f = f(o_att); ws.act.f = f(o_act); ws.side.f = f(o_sd);
    if (bf) { ws.xa.hi = h(o_xh); ws.xa.lo = h(o_xl); ws.att.hi = h(o_ah); ws.act.hi = h(o_gh); ws.side.hi = h(o_sh); }
    ws.qf = ws.base + o_q; ws.part_ctx = f(o_pc); ws.part_ml = f(o_pm);
    ws.z = f(o_z); ws.weight = f(o_wt); ws.row_scale = f(o_rs); ws.yexp = h(o_ye); ws.vec_act = f(o_va);
    ws.sel = i(o_sel); ws.pos = i(o_pos); ws.src = i(o_src); ws.n_tiles = i(o_nt); ws.tiles = reinterpret_cast<int4 *>(ws.base + o_tiles);
    ws.xperm = h(o_xp); ws.aperm = h(o_ap); ws.ids = f(o_ids); ws.logits = f(o_lg);
    LUMEN_CUDA(ctx, cudaMallocHost(&ws.h_ids, std::max<size_t>(M, 1) * sizeof(float)));
    ws.h_logits_elems = std::min<size_t>(M * V, (size_t)16 << 20);  // pinned staging up to 64 MB
    LUMEN_CUDA(ctx, cudaMallocHost(&ws.h_logits, std::max<size_t>(ws.h_logits_elems, 1) * sizeof(float)));
    ws.M = M;
    io = StepIo{ws.ids, ws.logits, ws.h_ids, ws.h_logits, ws.h_logits_elems};
    return LUMEN_OK;
}

LatentArgs lumen_decoder::latent_args(size_t l, lumen_kv_cache *c, size_t B, size_t S) const {
    const lumen_decoder_layer &k = lc[l];
    const LayerW &w = lw[l];
    LatentArgs a;
    a.B = B; a.S = S; a.H = k.heads; a.dim = k.dim; a.rot_dim = k.rot_dim; a.vdim = k.vdim; a.rank = k.kv_rank; a.rot_dims = k.rot_dims;
    a.pitch = w.pitch; a.max_seq = cfg.max_seq_len; a.dt = dt;
    a.u = ws.u; a.u_ld = w.proj_rows; a.u_kv = w.u_kv; a.u_gate = w.u_gate;
    a.latent_gain = w.latent_gain; a.eps = cfg.norm_eps; a.scale = k.scale; a.cos_t = w.cos_t; a.sin_t = w.sin_t;
    a.wuk = w.uk; a.wuv = w.uv; a.cache = c->k; a.d_len = c->d_len; a.past = c->len;
    a.qf = ws.qf; a.part_ctx = ws.part_ctx; a.part_ml = ws.part_ml;
    return a;
}

GroupedArgs lumen_decoder::grouped_args(size_t l, lumen_kv_cache *c, size_t B, size_t S) const {
    const lumen_decoder_layer &k = lc[l];
    const LayerW &w = lw[l];
    GroupedArgs a;
    a.B = B; a.S = S; a.H = k.heads; a.G = k.kv_heads; a.dim = k.dim; a.vdim = k.vdim; a.rot_dims = k.rot_dims; a.chunk = k.chunk;
    a.max_seq = cfg.max_seq_len; a.dt = dt;
    a.u = ws.u; a.u_ld = w.proj_rows; a.u_k = w.u_k; a.u_v = w.u_v; a.u_gate = w.u_gate; a.own_kv = k.kv_from < 0;
    a.q_gain = w.q_gain; a.k_gain = w.k_gain; a.sink = w.sink; a.eps = cfg.norm_eps; a.scale = k.scale; a.cos_t = w.cos_t; a.sin_t = w.sin_t;
    a.k = c->k; a.v = c->v; a.d_len = c->d_len; a.past = c->len;
    a.part_ctx = ws.part_ctx; a.part_ml = ws.part_ml;
    return a;
}

MlstmArgs lumen_decoder::mlstm_args(size_t l, lumen_kv_cache *c, size_t B, size_t S) const {
    const lumen_decoder_layer &k = lc[l];
    const LayerW &w = lw[l];
    MlstmArgs a;
    a.B = B; a.S = S; a.H = k.heads; a.dim = k.dim; a.vdim = k.vdim; a.cap = k.gate_cap; a.eps = cfg.norm_eps;
    a.u = ws.u; a.u_ld = w.main_rows; a.u_k = w.u_k; a.u_v = w.u_v; a.u_g = w.u_gate;
    a.z = ws.z; a.z_ld = 2 * k.heads; a.z_bias = w.z_bias; a.head_gain = w.head_gain;
    a.state = c->k; a.norm = c->v; a.mx = c->v + B * k.heads * k.dim; a.d_len = c->d_len; a.past = c->len;
    return a;
}

int lumen_decoder::pick_splits(size_t l, lumen_kv_cache *c, size_t B, size_t S) const {
    switch (lc[l].mixer) {
        case LUMEN_MIXER_LATENT: return latent_pick_splits(latent_args(l, c, B, S), c->len + S, ctx->num_sms);
        case LUMEN_MIXER_ATTENTION: return grouped_pick_splits(grouped_args(l, c, B, S), ctx->num_sms);
        default: return 1;
    }
}

MoeArgs lumen_decoder::moe_args(size_t l, size_t M) const {
    const lumen_decoder_layer &k = lc[l];
    const LayerW &w = lw[l];
    MoeArgs a;
    a.M = M; a.W = W; a.experts = k.experts; a.top = k.top; a.ff = k.expert_ff; a.shared_ff = k.shared_ff;
    a.limit = k.expert_limit; a.shared_limit = k.shared_limit; a.wdt = dt;
    a.z = ws.z; a.gate_up = w.gate_up; a.down = w.edown; a.shared_gate_up = w.sgate_up; a.shared_down = w.sdown;
    a.act = ws.vec_act; a.sel = ws.sel; a.y = ws.y;
    return a;
}

// One token of one sequence.  The residual alternates between two buffers: a product's input stage reads one and leaves the
// sum with the sublayer's normed output in the other.
int lumen_decoder::step_row(lumen_kv_cache **caches) {
    cudaStream_t s = ctx->stream;
    EmbedArgs e;
    e.ids = ws.ids; e.embed = embed; e.bigram = bigram; e.dt = dt; e.vocab = V; e.dim = W;
    e.buckets = cfg.bigram_buckets; e.mul_prev = cfg.bigram_mul_prev; e.mul_cur = cfg.bigram_mul_cur;
    e.d_len = caches[0]->d_len; e.last_tok = caches[0]->last_tok; e.x = ws.x[0]; e.scale = cfg.embed_scale;
    LUMEN_TRY(launch_embed(ctx, e, s));
    int cur = 0;
    Pending pend;
    // y = w . x, where x is the residual after the pending output (which is thereby settled), normed with norm_w if given
    auto from_residual = [&](const void *w, size_t N, float *out, StepFinish::Kind act, size_t layer, const float *norm_w = nullptr) -> int {
        GemvStepArgs g;
        g.res = ws.x[cur]; g.eps = cfg.norm_eps; g.w = w; g.wdt = dt; g.K = W; g.N = N; g.out = out; g.act = act; g.norm_w = norm_w;
        if (pend.y) {
            g.y = pend.y; g.gain = pend.gain; g.x_out = ws.x[cur ^ 1];
            cur ^= 1;
            pend = Pending();
        }
        if (act == StepFinish::kSideGate) {
            g.ids = ws.ids; g.table = side_embed + layer * cfg.side_dim * esz; g.table_ld = L * cfg.side_dim; g.table_rows = V;
        }
        return launch_gemv_step(ctx, g, s);
    };
    auto plain = [&](const float *a, const void *w, size_t K, const float *gain) -> int {
        GemvStepArgs g;
        g.res = a; g.w = w; g.wdt = dt; g.K = K; g.N = W; g.out = ws.y;
        pend.y = ws.y; pend.gain = gain;
        return launch_gemv_step(ctx, g, s);
    };
    for (size_t l = 0; l < L; ++l) {
        const lumen_decoder_layer &k = lc[l];
        const LayerW &w = lw[l];
        LUMEN_TRY(from_residual(w.proj, w.proj_rows, ws.u, StepFinish::kStore, l, w.pre1));
        if (k.mixer == LUMEN_MIXER_LATENT) {
            LatentArgs a = latent_args(l, caches[l], 1, 1);
            a.nsplit = pick_splits(l, caches[l], 1, 1);
            a.out = ws.att.f;
            LUMEN_TRY(launch_latent_absorb(ctx, a, true, s));
            LUMEN_TRY(latent_mma_usable(a) ? launch_latent_mma(ctx, a, s) : launch_latent_scores(ctx, a, s));
            LUMEN_TRY(launch_latent_value(ctx, a, s));
        } else if (k.mixer == LUMEN_MIXER_ATTENTION) {
            GroupedArgs a = grouped_args(l, caches[l], 1, 1);
            a.nsplit = pick_splits(l, caches[l], 1, 1);
            a.out = ws.att.f;
            LUMEN_TRY(launch_grouped_attention(ctx, a, a.own_kv, s));
        } else {
            MlstmArgs a = mlstm_args(l, caches[l], 1, 1);
            a.z = ws.u + w.main_rows;  // (one row: all projections are one product)
            a.out = ws.att.f;
            LUMEN_TRY(launch_mlstm_step(ctx, a, s));
        }
        LUMEN_TRY(plain(ws.att.f, w.o, k.heads * k.vdim, w.norm1));
        if (k.mlp_kind == LUMEN_MLP_DENSE) {
            LUMEN_TRY(from_residual(w.up, k.ff, ws.act.f, StepFinish::kGelu, l));
            LUMEN_TRY(plain(ws.act.f, w.down, k.ff, w.norm2));
        } else if (k.mlp_kind == LUMEN_MLP_GATED_GELU) {
            LUMEN_TRY(from_residual(w.up, k.ff, ws.act.f, StepFinish::kGated, l, w.pre2));
            LUMEN_TRY(plain(ws.act.f, w.down, k.ff, w.norm2));
        } else if (k.mlp_kind == LUMEN_MLP_MOE) {
            LUMEN_TRY(from_residual(w.router, k.experts, ws.z, StepFinish::kStore, l));
            MoeArgs m = moe_args(l, 1);
            m.x = ws.x[cur];
            LUMEN_TRY(launch_moe_vec(ctx, m, s));
            pend.y = ws.y; pend.gain = w.norm2;
        }
        if (cfg.side_dim) {
            LUMEN_TRY(from_residual(w.side_gate, cfg.side_dim, ws.side.f, StepFinish::kSideGate, l));
            LUMEN_TRY(plain(ws.side.f, w.side_proj, cfg.side_dim, w.side_norm));
        }
    }
    LUMEN_TRY(from_residual(head, V, ws.logits, StepFinish::kStore, 0, final_gain));
    return launch_advance(ctx, caches[0]->d_len, L, ws.ids, caches[0]->last_tok, 1, 1, s);
}

// c = a . w^T, then `fin` (null: c is the result).  `pair`: multiply the hi/lo pair of the activations instead of hi alone.
int lumen_decoder::product(const Act &a, size_t lda, const void *w, size_t M, size_t K, size_t N, float *c, const StepFinish *fin, bool pair) {
    cudaStream_t s = ctx->stream;
    if (on_tensor_cores(M, K)) {
        GemmBf16Args g;
        g.a_hi = a.hi; g.a_lo = pair ? a.lo : nullptr; g.M = M; g.K = K; g.lda = lda; g.N = N;
        g.w = static_cast<const __nv_bfloat16 *>(w); g.c = c; g.fin = fin;
        return launch_gemm_bf16(ctx, g, s);
    }
    if (M <= 8 && M * K * 4 <= 200 * 1024) {
        GemvArgs g;
        g.x = a.f; g.w = w; g.wdt = dt; g.y = c; g.M = (int)M; g.K = K; g.N = N; g.ldy = N;
        LUMEN_TRY(launch_gemv_nk(ctx, g, s));
    } else {
        LUMEN_TRY(launch_gemm_simt(ctx, a.f, w, dt, c, M, K, N, nullptr, s));
    }
    return fin ? launch_step_finish(ctx, c, 1, M, N, *fin, s) : LUMEN_OK;
}

int lumen_decoder::mix_rows(size_t l, lumen_kv_cache *c, size_t B, size_t S) {
    cudaStream_t s = ctx->stream;
    const lumen_decoder_layer &k = lc[l];
    const LayerW &w = lw[l];
    const size_t M = B * S, av = k.heads * k.vdim;
    auto output = [&](auto &a) {
        if (on_tensor_cores(M, av)) a.out_hi = ws.att.hi;
        else a.out = ws.att.f;
    };
    if (k.mixer == LUMEN_MIXER_MLSTM) {
        MlstmArgs a = mlstm_args(l, c, B, S);
        output(a);
        const char *gates = w.proj + w.main_rows * W * esz;
        LUMEN_TRY(product(ws.xa, W, gates, M, W, 2 * k.heads, ws.z, nullptr, true));
        if (on_tensor_cores(M, W) && mlstm_chunked_usable(a)) {
            GemmBf16Args g;
            g.a_hi = ws.xa.hi; g.M = M; g.K = W; g.w = reinterpret_cast<const __nv_bfloat16 *>(w.proj); g.N = w.main_rows;
            g.out16 = reinterpret_cast<__nv_bfloat16 *>(ws.u); g.ld16 = w.main_rows; g.epi = GemmBf16Args::kBf16;
            LUMEN_TRY(launch_gemm_bf16(ctx, g, s));
            a.u16 = g.out16;
            return launch_mlstm_chunked(ctx, a, s);
        }
        LUMEN_TRY(product(ws.xa, W, w.proj, M, W, w.main_rows, ws.u, nullptr));
        return launch_mlstm_step(ctx, a, s);
    }
    LUMEN_TRY(product(ws.xa, W, w.proj, M, W, w.proj_rows, ws.u, nullptr));
    if (k.mixer == LUMEN_MIXER_ATTENTION) {
        GroupedArgs a = grouped_args(l, c, B, S);
        output(a);
        if (grouped_prefill_usable(a)) return launch_grouped_prefill(ctx, a, s);
        a.nsplit = pick_splits(l, c, B, S);
        const bool append = a.own_kv && S == 1;
        if (!append) LUMEN_TRY(launch_grouped_append(ctx, a, nullptr, 0, 0, s));
        return launch_grouped_attention(ctx, a, append, s);
    }
    LatentArgs a = latent_args(l, c, B, S);
    output(a);
    if (latent_prefill_usable(a)) {
        LUMEN_TRY(launch_latent_append(ctx, a, s));
        return launch_latent_prefill(ctx, a, s);
    }
    a.nsplit = pick_splits(l, c, B, S);
    LUMEN_TRY(launch_latent_absorb(ctx, a, true, s));
    LUMEN_TRY(latent_mma_usable(a) ? launch_latent_mma(ctx, a, s) : launch_latent_scores(ctx, a, s));
    return launch_latent_value(ctx, a, s);
}

// S positions of B sequences.
int lumen_decoder::step_rows(size_t B, size_t S, lumen_kv_cache **caches, bool last_only) {
    cudaStream_t s = ctx->stream;
    const size_t M = B * S;
    const bool bf = dt == LUMEN_BF16;
    EmbedArgs e;
    e.ids = ws.ids; e.embed = embed; e.bigram = bigram; e.dt = dt; e.B = B; e.S = S; e.vocab = V; e.dim = W;
    e.buckets = cfg.bigram_buckets; e.mul_prev = cfg.bigram_mul_prev; e.mul_cur = cfg.bigram_mul_cur;
    e.d_len = caches[0]->d_len; e.last_tok = caches[0]->last_tok; e.x = ws.x[0]; e.hi = ws.xa.hi; e.scale = cfg.embed_scale;
    if (norms_before()) {
        e.norm_w = lw[0].pre1; e.eps = cfg.norm_eps;
        if (!on_tensor_cores(M, W)) e.out = ws.xa.f;
        if (lc[0].mixer == LUMEN_MIXER_MLSTM) e.lo = ws.xa.lo;  // (its gates read a pair)
    }
    LUMEN_TRY(launch_embed(ctx, e, s));
    // What the products of this step read of an activation: bf16 on the tensor cores, f32 otherwise.
    auto target = [&](StepFinish &f, const Act &a, size_t K) {
        if (on_tensor_cores(M, K)) f.hi = a.hi;
        else f.out = a.f;
    };
    // next: gain of the norm before the next sublayer (null: it reads the residual); pair: it reads a hi/lo pair
    auto norm_add = [&](const float *gain, bool pair = false, const float *next = nullptr) {
        StepFinish f;
        f.kind = StepFinish::kNormAdd; f.x = ws.x[0]; f.gain = gain; f.eps = cfg.norm_eps; f.hi = ws.xa.hi; f.next_gain = next;
        if (pair) f.lo = ws.xa.lo;
        if (next && !on_tensor_cores(M, W)) f.out = ws.xa.f;
        return f;
    };
    auto is_mlstm = [&](size_t l) { return l < L && lc[l].mixer == LUMEN_MIXER_MLSTM; };
    // Products whose activation is applied in the epilogue: enough rows that K is not split.
    const bool epilogue = M > 128;
    for (size_t l = 0; l < L; ++l) {
        const lumen_decoder_layer &k = lc[l];
        const LayerW &w = lw[l];
        const size_t av = k.heads * k.vdim;
        LUMEN_TRY(mix_rows(l, caches[l], B, S));
        // what comes next and what it reads: the router and the gates of a matrix memory read pairs
        const bool last = k.mlp_kind == LUMEN_MLP_NONE;  // the mixer is the layer's last sublayer
        const float *after = l + 1 < L ? lw[l + 1].pre1 : nullptr;
        StepFinish f1 = norm_add(w.norm1, k.mlp_kind == LUMEN_MLP_MOE || (last && is_mlstm(l + 1)), last ? after : w.pre2);
        LUMEN_TRY(product(ws.att, av, w.o, M, av, W, ws.y, &f1));
        if (k.mlp_kind == LUMEN_MLP_DENSE) {
            if (epilogue && on_tensor_cores(M, W) && on_tensor_cores(M, k.ff)) {
                GemmBf16Args g;
                g.a_hi = ws.xa.hi; g.M = M; g.K = W; g.w = reinterpret_cast<const __nv_bfloat16 *>(w.up); g.N = k.ff;
                g.out16 = ws.act.hi; g.ld16 = k.ff; g.epi = GemmBf16Args::kGelu;
                LUMEN_TRY(launch_gemm_bf16(ctx, g, s));
            } else {
                StepFinish fa;
                fa.kind = StepFinish::kGelu;
                target(fa, ws.act, k.ff);
                LUMEN_TRY(product(ws.xa, W, w.up, M, W, k.ff, ws.c, &fa));
            }
            StepFinish f2 = norm_add(w.norm2, is_mlstm(l + 1), after);
            LUMEN_TRY(product(ws.act, k.ff, w.down, M, k.ff, W, ws.y, &f2));
        } else if (k.mlp_kind == LUMEN_MLP_GATED_GELU) {
            if (epilogue && on_tensor_cores(M, W) && on_tensor_cores(M, k.ff)) {
                GemmBf16Args g;
                g.a_hi = ws.xa.hi; g.M = M; g.K = W; g.w = reinterpret_cast<const __nv_bfloat16 *>(w.up); g.N = gated_rows(k.ff);
                g.ff = k.ff; g.out16 = ws.act.hi; g.ld16 = k.ff; g.epi = GemmBf16Args::kGatedGelu;
                LUMEN_TRY(launch_gemm_bf16(ctx, g, s));
            } else {
                StepFinish fa;
                fa.kind = StepFinish::kGated; fa.glu = StepFinish::kGeluTanh; fa.ff = k.ff;
                target(fa, ws.act, k.ff);
                LUMEN_TRY(product(ws.xa, W, w.up, M, W, gated_rows(k.ff), ws.c, &fa));
            }
            StepFinish f2 = norm_add(w.norm2, is_mlstm(l + 1), after);
            LUMEN_TRY(product(ws.act, k.ff, w.down, M, k.ff, W, ws.y, &f2));
        } else if (k.mlp_kind == LUMEN_MLP_MOE) {
            LUMEN_TRY(product(ws.xa, W, w.router, M, W, k.experts, ws.z, nullptr, true));
            StepFinish f2 = norm_add(w.norm2, is_mlstm(l + 1), after);
            if (on_tensor_cores(M, W) && on_tensor_cores(M, k.expert_ff)) {
                MoeGroupArgs ga;
                ga.M = M; ga.experts = k.experts; ga.top = k.top; ga.z = ws.z; ga.sel = ws.sel; ga.pos = ws.pos; ga.src = ws.src;
                ga.weight = ws.weight; ga.row_scale = ws.row_scale; ga.tiles = ws.tiles; ga.n_tiles = ws.n_tiles;
                LUMEN_TRY(launch_moe_group(ctx, ga, s));
                LUMEN_TRY(launch_gather_rows(ctx, ws.xa.hi, ws.src, ws.xperm, M * k.top, W, s));
                GemmBf16Args g;
                g.a_hi = ws.xperm; g.M = M * k.top; g.K = W; g.w = reinterpret_cast<const __nv_bfloat16 *>(w.gate_up);
                g.N = gated_rows(k.expert_ff); g.w_groups = k.experts; g.tiles = ws.tiles; g.n_tiles = ws.n_tiles;
                g.max_tiles = moe_max_tiles(M, k.experts, k.top); g.row_scale = ws.row_scale; g.limit = k.expert_limit; g.ff = k.expert_ff;
                g.out16 = ws.aperm; g.ld16 = k.expert_ff; g.epi = GemmBf16Args::kGated;
                LUMEN_TRY(launch_gemm_bf16(ctx, g, s));
                GemmBf16Args d;
                d.a_hi = ws.aperm; d.M = M * k.top; d.K = k.expert_ff; d.w = reinterpret_cast<const __nv_bfloat16 *>(w.edown);
                d.N = W; d.w_groups = k.experts; d.tiles = ws.tiles; d.n_tiles = ws.n_tiles; d.max_tiles = g.max_tiles; d.out16 = ws.yexp; d.ld16 = W;
                d.epi = GemmBf16Args::kBf16;
                LUMEN_TRY(launch_gemm_bf16(ctx, d, s));
                f2.gather_src = ws.yexp; f2.gather_idx = ws.pos; f2.gather_n = (int)k.top;
                if (k.shared_ff) {
                    const bool tc = on_tensor_cores(M, k.shared_ff);
                    if (epilogue && tc) {
                        GemmBf16Args sg;
                        sg.a_hi = ws.xa.hi; sg.M = M; sg.K = W; sg.w = reinterpret_cast<const __nv_bfloat16 *>(w.sgate_up);
                        sg.N = gated_rows(k.shared_ff); sg.limit = k.shared_limit; sg.ff = k.shared_ff; sg.out16 = ws.act.hi; sg.ld16 = k.shared_ff;
                        sg.epi = GemmBf16Args::kGated;
                        LUMEN_TRY(launch_gemm_bf16(ctx, sg, s));
                    } else {
                        StepFinish fg;
                        fg.kind = StepFinish::kGated; fg.limit = k.shared_limit; fg.ff = k.shared_ff;
                        target(fg, ws.act, k.shared_ff);
                        LUMEN_TRY(product(ws.xa, W, w.sgate_up, M, W, gated_rows(k.shared_ff), ws.c, &fg));
                    }
                    LUMEN_TRY(product(ws.act, k.shared_ff, w.sdown, M, k.shared_ff, W, ws.y, &f2));
                } else {
                    LUMEN_TRY(launch_step_finish(ctx, nullptr, 0, M, W, f2, s));
                }
            } else {
                MoeArgs m = moe_args(l, M);
                m.x = ws.x[0];
                LUMEN_TRY(launch_moe_vec(ctx, m, s));
                LUMEN_TRY(launch_step_finish(ctx, ws.y, 1, M, W, f2, s));
            }
        }
        if (cfg.side_dim) {
            StepFinish fs;
            fs.kind = StepFinish::kSideGate; fs.ids = ws.ids; fs.table = side_embed + l * cfg.side_dim * esz; fs.table_dt = dt;
            fs.table_ld = L * cfg.side_dim; fs.table_rows = V;
            target(fs, ws.side, cfg.side_dim);
            LUMEN_TRY(product(ws.xa, W, w.side_gate, M, W, cfg.side_dim, ws.c, &fs));
            StepFinish f3 = norm_add(w.side_norm, is_mlstm(l + 1), after);
            LUMEN_TRY(product(ws.side, cfg.side_dim, w.side_proj, M, cfg.side_dim, W, ws.y, &f3));
        }
    }
    const float *xin = ws.x[0];
    size_t rows = M;
    if (last_only && S > 1) {
        LUMEN_CUDA(ctx, cudaMemcpy2DAsync(ws.last_x, W * 4, ws.x[0] + (S - 1) * W, S * W * 4, W * 4, B, cudaMemcpyDeviceToDevice, s));
        xin = ws.last_x;
        rows = B;
    }
    if (rows <= (bf && on_tensor_cores(2, W) ? 1 : 8) && rows * W * 4 <= 200 * 1024) {
        GemvArgs g;
        g.x = xin; g.w = head; g.wdt = dt; g.y = ws.logits; g.M = (int)rows; g.K = W; g.N = V; g.ldy = V; g.norm_w = final_gain; g.norm_eps = cfg.norm_eps;
        LUMEN_TRY(launch_gemv_nk(ctx, g, s));
    } else {
        LUMEN_TRY(launch_rmsnorm(ctx, xin, final_gain, cfg.norm_eps, ws.nx, rows, W, s));
        Act n;
        n.f = ws.nx;
        if (on_tensor_cores(rows, W)) {
            n.hi = ws.xa.hi; n.lo = ws.xa.lo;
            LUMEN_TRY(launch_split_bf16(ctx, ws.nx, n.hi, n.lo, rows * W, s));
        }
        LUMEN_TRY(product(n, W, head, rows, W, V, ws.logits, nullptr, true));
    }
    return launch_advance(ctx, caches[0]->d_len, L, ws.ids, caches[0]->last_tok, B, S, s);
}

int lumen_decoder::run_forward(size_t b, size_t s, lumen_kv_cache **caches, bool last_only) {
    int rc;
    if (s == 1) {
        // every launch of the step reads the position from the device; only the pieces of the context are baked in
        // (a context picks the same piece counts for all layers of one geometry, so their combination grows with the context)
        unsigned key = 0;
        for (size_t l = 0; l < L; ++l) key = key * 7 + (unsigned)pick_splits(l, caches[l], b, 1);
        const bool one = b == 1 && W * 4 <= 200 * 1024;
        rc = run_graphed(std::make_tuple(b, (int)key, (const void *)caches[0]->k),
                         [&] {
                             ctx->pdl = one;
                             const int r = one ? step_row(caches) : step_rows(b, 1, caches, last_only);
                             ctx->pdl = false;
                             return r;
                         });
    } else {
        rc = step_rows(b, s, caches, last_only);
    }
    if (rc == LUMEN_OK)
        for (size_t l = 0; l < L; ++l) caches[l]->len += s;
    return rc;
}

}  // namespace

extern "C" int lumen_decoder_new(lumen_ctx *ctx, const lumen_decoder_config *cfg, lumen_model **out) {
    if (!ctx || !cfg || !out || (cfg->num_layers && !cfg->layers)) return set_error(ctx, LUMEN_ERR_INVALID, "decoder_new: null argument");
    if (cfg->weight_dtype != LUMEN_F32 && cfg->weight_dtype != LUMEN_BF16) return set_error(ctx, LUMEN_ERR_DTYPE, "weight_dtype %d", (int)cfg->weight_dtype);
    if (ctx->tp_size > 1) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "models given as a list of layers run on one GPU (tp_size %d)", ctx->tp_size);
    if (!cfg->vocab_size || !cfg->width || !cfg->max_seq_len || !cfg->num_layers) return set_error(ctx, LUMEN_ERR_SHAPE, "decoder_new: empty model");
    for (size_t l = 0; l < cfg->num_layers; ++l) {
        const lumen_decoder_layer &k = cfg->layers[l];
        if (!k.heads || !k.dim || !k.vdim || k.rot_dims % 2) return set_error(ctx, LUMEN_ERR_SHAPE, "layer %zu: mixer sizes", l);
        if (k.mixer == LUMEN_MIXER_LATENT) {
            if (!k.kv_rank || k.rot_dims > k.rot_dim) return set_error(ctx, LUMEN_ERR_SHAPE, "layer %zu: latent attention sizes", l);
        } else if (k.mixer == LUMEN_MIXER_ATTENTION) {
            if (!k.kv_heads || k.heads % k.kv_heads || k.rot_dims > k.dim) return set_error(ctx, LUMEN_ERR_SHAPE, "layer %zu: attention sizes", l);
            if (std::max(k.dim, k.vdim) > kGroupedMaxDim) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "layer %zu: heads of %zu / %zu numbers (at most %zu)", l, k.dim, k.vdim, kGroupedMaxDim);
            if (k.kv_from >= 0) {
                const lumen_decoder_layer *j = (size_t)k.kv_from < l ? &cfg->layers[k.kv_from] : nullptr;
                if (!j || j->mixer != LUMEN_MIXER_ATTENTION || j->kv_from >= 0 || j->kv_heads != k.kv_heads || j->dim != k.dim || j->vdim != k.vdim)
                    return set_error(ctx, LUMEN_ERR_SHAPE, "layer %zu: keys and values of layer %d", l, k.kv_from);
            }
        } else if (k.mixer != LUMEN_MIXER_MLSTM || !(k.gate_cap > 0.f)) {
            return set_error(ctx, LUMEN_ERR_SHAPE, "layer %zu: mixer %d", l, k.mixer);
        }
        if (k.kv_rank > 1024) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "layer %zu: latent of %zu numbers (at most 1024)", l, k.kv_rank);
        if (k.mlp_kind == LUMEN_MLP_DENSE || k.mlp_kind == LUMEN_MLP_GATED_GELU ? !k.ff : k.mlp_kind == LUMEN_MLP_MOE ? (!k.experts || !k.top || k.top > k.experts || !k.expert_ff) : k.mlp_kind != LUMEN_MLP_NONE)
            return set_error(ctx, LUMEN_ERR_SHAPE, "layer %zu: feed-forward sizes", l);
        if (k.mlp_kind == LUMEN_MLP_MOE && k.experts > 1536) return set_error(ctx, LUMEN_ERR_UNSUPPORTED, "layer %zu: %zu experts (at most 1536)", l, k.experts);
    }
    if (cfg->norms != LUMEN_NORM_OUTPUT && cfg->norms != LUMEN_NORM_BOTH) return set_error(ctx, LUMEN_ERR_INVALID, "decoder_new: norms %d", cfg->norms);
    auto *m = new lumen_decoder();
    m->ctx = ctx;
    m->cfg = *cfg;
    m->lc.assign(cfg->layers, cfg->layers + cfg->num_layers);
    m->cfg.layers = nullptr;
    m->V = cfg->vocab_size; m->W = cfg->width; m->L = cfg->num_layers; m->dt = cfg->weight_dtype;
    m->esz = cfg->weight_dtype == LUMEN_F32 ? 4 : 2;
    m->lw.resize(m->L);
    const char *ng = getenv("LUMEN_NO_GRAPH");
    m->use_graph = !(ng && ng[0] == '1');
    const int rc = m->build();
    if (rc != LUMEN_OK) {
        delete m;
        return rc;
    }
    *out = m;
    return LUMEN_OK;
}
