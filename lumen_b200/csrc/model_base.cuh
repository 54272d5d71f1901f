// What every language model behind the C ABI shares: the host side of a forward step (id checks, pinned staging of ids and
// logits, sampling on the device), the store of captured decode graphs, and the upload of parameters.  A model derives from
// lumen_model and supplies its workspace, its cache checks and the step itself; the entry points lumen_model_* (and the
// lumen_llama_* ones, which keep the reference's names) call through it.
#pragma once

#include <functional>
#include <map>
#include <tuple>

#include "common.cuh"

namespace lumen {

inline size_t align_up(size_t v, size_t a) { return (v + a - 1) / a * a; }

// Buffers a step reads its ids from and leaves its logits in; owned by the model's workspace.
struct StepIo {
    float *ids = nullptr, *logits = nullptr;      // device
    float *h_ids = nullptr, *h_logits = nullptr;  // pinned host staging
    size_t h_logits_elems = 0;
};

// Copies the [rows x ncols] block starting at column col0 of a row-major host matrix with `cols_total` columns into a dense
// device matrix of dtype dst_dt, converting between f32 and bf16 when needed.
int upload_block(lumen_ctx *ctx, void *dst, lumen_dtype dst_dt, const void *src_host, lumen_dtype src_dt, size_t rows,
                 size_t cols_total, size_t col0, size_t ncols);

// Device slab that the layer caches of one init_kv_caches call share (freed with the last of them).
lumen_storage *new_cache_slab(lumen_ctx *ctx, size_t bytes, int *rc);

// Ids of a step must be below the vocabulary (src/layers/basic/embedding.rs:50-56 of the reference); checked before a launch.
int check_ids(lumen_ctx *ctx, const float *ids_host, size_t n, size_t vocab);

}  // namespace lumen

struct lumen_model {
    lumen_ctx *ctx = nullptr;
    size_t V = 0;          // vocabulary
    size_t L = 0;          // layers, one cache each
    size_t n_expected = 0; // parameters that must be set before the first step
    std::map<std::string, bool> is_set;
    lumen::StepIo io;

    virtual ~lumen_model() {}
    virtual int set_param(const char *name, const void *host_data, const size_t *shape, int ndim, lumen_dtype dtype) = 0;
    virtual int init_kv_caches(size_t batch, lumen_kv_cache **out) = 0;
    virtual int check_caches(size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches) = 0;
    virtual int ensure_workspace(size_t rows) = 0;  // sets io
    // One forward over io.ids[b * s]; logits in io.logits ([b * s, V], or [b, V] with last_only and s > 1).
    virtual int run_forward(size_t b, size_t s, lumen_kv_cache **caches, bool last_only) = 0;
    virtual size_t weight_bytes() const = 0;

    int ready();
    int forward_host(const float *ids_host, size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches, float *logits_host, bool last_only);
    int forward_sample(const float *ids_host, size_t s, lumen_kv_cache **caches, size_t n_caches, const lumen_sample_params *sp, int32_t *token_out);
    int forward_device(const float *ids_dev, size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches, float *logits_dev);

    // Decode steps: the first call with a key runs `enqueue` eagerly, the second captures it, later ones replay the graph.
    // The key names everything that is baked into the launches (batch, split count, cache address).
    using GraphKey = std::tuple<size_t, int, const void *>;
    bool use_graph = true;
    int run_graphed(const GraphKey &key, const std::function<int()> &enqueue);
    void drop_graphs();

  private:
    struct Captured {
        int eager_runs = 0;
        cudaGraphExec_t exec = nullptr;
        unsigned long long nodes = 0;
    };
    std::map<GraphKey, Captured> graphs_;
};
