// The model-independent half of a step and the entry points lumen_model_*; see model_base.cuh.
#include "model_base.cuh"

#include <algorithm>

using namespace lumen;

namespace lumen {
namespace {

__global__ void f32_to_bf16_kernel(const float *in, __nv_bfloat16 *out, size_t n) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = __float2bfloat16_rn(in[i]);
}
__global__ void bf16_to_f32_kernel(const __nv_bfloat16 *in, float *out, size_t n) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = __bfloat162float(in[i]);
}

}  // namespace

int upload_block(lumen_ctx *ctx, void *dst, lumen_dtype dst_dt, const void *src_host, lumen_dtype src_dt, size_t rows,
                 size_t cols_total, size_t col0, size_t ncols) {
    if (rows == 0 || ncols == 0) return LUMEN_OK;
    const size_t se = src_dt == LUMEN_F32 ? 4 : 2;
    const char *src = static_cast<const char *>(src_host) + col0 * se;
    cudaStream_t s = ctx->stream;
    if (src_dt == dst_dt) {
        LUMEN_CUDA(ctx, cudaMemcpy2DAsync(dst, ncols * se, src, cols_total * se, ncols * se, rows, cudaMemcpyHostToDevice, s));
        LUMEN_CUDA(ctx, cudaStreamSynchronize(s));
        return LUMEN_OK;
    }
    // Convert in row chunks to bound the staging buffer.
    const size_t chunk_rows = std::max<size_t>(1, ((size_t)64 << 20) / (ncols * se));
    void *tmp = nullptr;
    LUMEN_CUDA(ctx, cudaMalloc(&tmp, std::min(rows, chunk_rows) * ncols * se));
    const size_t de = dst_dt == LUMEN_F32 ? 4 : 2;
    int rc = LUMEN_OK;
    for (size_t r0 = 0; r0 < rows && rc == LUMEN_OK; r0 += chunk_rows) {
        const size_t nr = std::min(chunk_rows, rows - r0), n = nr * ncols;
        cudaError_t e = cudaMemcpy2DAsync(tmp, ncols * se, src + r0 * cols_total * se, cols_total * se, ncols * se, nr,
                                          cudaMemcpyHostToDevice, s);
        if (e != cudaSuccess) { rc = cuda_fail(ctx, e, "cudaMemcpy2DAsync"); break; }
        char *d = static_cast<char *>(dst) + r0 * ncols * de;
        if (dst_dt == LUMEN_BF16)
            f32_to_bf16_kernel<<<(unsigned)((n + 255) / 256), 256, 0, s>>>((const float *)tmp, (__nv_bfloat16 *)d, n);
        else
            bf16_to_f32_kernel<<<(unsigned)((n + 255) / 256), 256, 0, s>>>((const __nv_bfloat16 *)tmp, (float *)d, n);
        e = cudaStreamSynchronize(s);
        if (e != cudaSuccess) rc = cuda_fail(ctx, e, "convert upload");
    }
    cudaFree(tmp);
    return rc;
}

lumen_storage *new_cache_slab(lumen_ctx *ctx, size_t bytes, int *rc) {
    auto *slab = new lumen_storage();
    slab->ctx = ctx;
    slab->bytes = bytes;
    slab->refs = 0;
    cudaError_t e = cudaMalloc(&slab->ptr, std::max<size_t>(bytes, 256));
    if (e == cudaSuccess) {
        e = cudaMemsetAsync(slab->ptr, 0, bytes, ctx->stream);  // Array4::zeros, self_attention.rs:35-36
        if (e != cudaSuccess) cudaFree(slab->ptr);
    }
    if (e != cudaSuccess) {
        delete slab;
        *rc = cuda_fail(ctx, e, "cudaMalloc(kv slab)");
        return nullptr;
    }
    *rc = LUMEN_OK;
    return slab;
}

int check_ids(lumen_ctx *ctx, const float *ids_host, size_t n, size_t vocab) {
    for (size_t i = 0; i < n; ++i) {
        const float f = ids_host[i];
        if (f >= (float)vocab && f == f) return set_error(ctx, LUMEN_ERR_EMBED_RANGE, "Embedding index out of bounds: %.0f >= %zu", (double)f, vocab);
    }
    return LUMEN_OK;
}

}  // namespace lumen

void lumen_model::drop_graphs() {
    for (auto &kv : graphs_)
        if (kv.second.exec) cudaGraphExecDestroy(kv.second.exec);
    graphs_.clear();
}

int lumen_model::run_graphed(const GraphKey &key, const std::function<int()> &enqueue) {
    if (!use_graph) return enqueue();
    Captured &c = graphs_[key];
    if (!c.exec && c.eager_runs++ >= 1) {
        cudaGraph_t graph = nullptr;
        const unsigned long long before = ctx->launches;
        LUMEN_CUDA(ctx, cudaStreamBeginCapture(ctx->stream, cudaStreamCaptureModeThreadLocal));
        const int rc = enqueue();
        cudaError_t e = cudaStreamEndCapture(ctx->stream, &graph);
        c.nodes = ctx->launches - before;  // captured, not run
        ctx->launches = before;
        if (rc != LUMEN_OK) {
            if (graph) cudaGraphDestroy(graph);
            return rc;
        }
        if (e != cudaSuccess) return cuda_fail(ctx, e, "cudaStreamEndCapture");
        e = cudaGraphInstantiate(&c.exec, graph, 0);
        cudaGraphDestroy(graph);
        if (e != cudaSuccess) {
            c.exec = nullptr;
            return cuda_fail(ctx, e, "cudaGraphInstantiate");
        }
    }
    if (!c.exec) return enqueue();
    LUMEN_CUDA(ctx, cudaGraphLaunch(c.exec, ctx->stream));
    ctx->launches += c.nodes;
    return LUMEN_OK;
}

int lumen_model::ready() {
    if (is_set.size() < n_expected) return set_error(ctx, LUMEN_ERR_MISSING_PARAM, "%zu of %zu parameters set", is_set.size(), n_expected);
    return LUMEN_OK;
}

int lumen_model::forward_host(const float *ids_host, size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches, float *logits_host,
                              bool last_only) {
    if (!ids_host || !logits_host) return LUMEN_ERR_INVALID;
    LUMEN_TRY(ready());
    const size_t M = b * s;
    if (M == 0) return LUMEN_OK;
    LUMEN_TRY(check_caches(b, s, caches, n_caches));
    LUMEN_TRY(check_ids(ctx, ids_host, M, V));
    LUMEN_TRY(ensure_workspace(M));
    // The pinned staging buffers are reused every step: wait for the previous step's copies first.
    LUMEN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    memcpy(io.h_ids, ids_host, M * sizeof(float));
    LUMEN_CUDA(ctx, cudaMemcpyAsync(io.ids, io.h_ids, M * sizeof(float), cudaMemcpyHostToDevice, ctx->stream));
    LUMEN_TRY(run_forward(b, s, caches, last_only));
    const size_t rows = (last_only && s > 1) ? b : M;
    const size_t n = rows * V;
    if (n <= io.h_logits_elems) {
        LUMEN_CUDA(ctx, cudaMemcpyAsync(io.h_logits, io.logits, n * 4, cudaMemcpyDeviceToHost, ctx->stream));
        LUMEN_TRY(check_device_status(ctx));
        memcpy(logits_host, io.h_logits, n * 4);
    } else {
        LUMEN_CUDA(ctx, cudaMemcpyAsync(logits_host, io.logits, n * 4, cudaMemcpyDeviceToHost, ctx->stream));
        LUMEN_TRY(check_device_status(ctx));
    }
    return LUMEN_OK;
}

int lumen_model::forward_sample(const float *ids_host, size_t s, lumen_kv_cache **caches, size_t n_caches, const lumen_sample_params *sp,
                                int32_t *token_out) {
    if (!ids_host || !sp || !token_out || (sp->n_recent && !sp->recent_tokens)) return LUMEN_ERR_INVALID;
    LUMEN_TRY(ready());
    if (s == 0) return set_error(ctx, LUMEN_ERR_SHAPE, "forward_sample: empty input");
    LUMEN_TRY(check_caches(1, s, caches, n_caches));
    LUMEN_TRY(check_ids(ctx, ids_host, s, V));
    LUMEN_TRY(ensure_workspace(s));
    LUMEN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));  // the pinned staging buffer is reused every step
    memcpy(io.h_ids, ids_host, s * sizeof(float));
    LUMEN_CUDA(ctx, cudaMemcpyAsync(io.ids, io.h_ids, s * sizeof(float), cudaMemcpyHostToDevice, ctx->stream));
    LUMEN_TRY(run_forward(1, s, caches, true));  // last position's logits in io.logits[V]
    int *token_dev = reinterpret_cast<int *>(io.ids);  // the id buffer is free again once the forward is enqueued behind it
    LUMEN_TRY(launch_sample_top_p(ctx, io.logits, V, sp->temperature, sp->top_p, sp->repetition_penalty, sp->recent_tokens, sp->n_recent,
                                  sp->uniform, token_dev, ctx->stream));
    LUMEN_CUDA(ctx, cudaMemcpyAsync(io.h_ids, token_dev, sizeof(int), cudaMemcpyDeviceToHost, ctx->stream));
    LUMEN_TRY(check_device_status(ctx));
    memcpy(token_out, io.h_ids, sizeof(int));
    return LUMEN_OK;
}

int lumen_model::forward_device(const float *ids_dev, size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches, float *logits_dev) {
    if (!ids_dev || !logits_dev) return LUMEN_ERR_INVALID;
    LUMEN_TRY(ready());
    const size_t M = b * s;
    if (M == 0) return LUMEN_OK;
    LUMEN_TRY(check_caches(b, s, caches, n_caches));
    LUMEN_TRY(ensure_workspace(M));
    LUMEN_CUDA(ctx, cudaMemcpyAsync(io.ids, ids_dev, M * sizeof(float), cudaMemcpyDeviceToDevice, ctx->stream));
    LUMEN_TRY(run_forward(b, s, caches, false));
    LUMEN_CUDA(ctx, cudaMemcpyAsync(logits_dev, io.logits, M * V * sizeof(float), cudaMemcpyDeviceToDevice, ctx->stream));
    return LUMEN_OK;
}

extern "C" {

int lumen_model_set_param(lumen_model *m, const char *name, const void *host_data, const size_t *shape, int ndim, lumen_dtype dtype) {
    if (!m || !name || !host_data || !shape) return LUMEN_ERR_INVALID;
    if (dtype != LUMEN_F32 && dtype != LUMEN_BF16) return set_error(m->ctx, LUMEN_ERR_DTYPE, "set_param: dtype %d", (int)dtype);
    return m->set_param(name, host_data, shape, ndim, dtype);
}

int lumen_model_init_kv_caches(lumen_model *m, size_t batch, lumen_kv_cache **caches_out) {
    if (!m || !caches_out) return LUMEN_ERR_INVALID;
    return m->init_kv_caches(batch, caches_out);
}

int lumen_model_reset_kv_caches(lumen_model *m, lumen_kv_cache **caches, size_t n_caches) {
    if (!m || (!caches && n_caches)) return LUMEN_ERR_INVALID;
    for (size_t i = 0; i < n_caches; ++i) LUMEN_TRY(lumen_kv_reset(caches[i]));
    return LUMEN_OK;
}

int lumen_model_forward(lumen_model *m, const float *ids_host, size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches,
                        float *logits_host) {
    return m ? m->forward_host(ids_host, b, s, caches, n_caches, logits_host, false) : LUMEN_ERR_INVALID;
}

int lumen_model_forward_last(lumen_model *m, const float *ids_host, size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches,
                             float *logits_host) {
    return m ? m->forward_host(ids_host, b, s, caches, n_caches, logits_host, true) : LUMEN_ERR_INVALID;
}

int lumen_model_forward_device(lumen_model *m, const float *ids_dev, size_t b, size_t s, lumen_kv_cache **caches, size_t n_caches,
                               float *logits_dev) {
    return m ? m->forward_device(ids_dev, b, s, caches, n_caches, logits_dev) : LUMEN_ERR_INVALID;
}

int lumen_model_forward_sample(lumen_model *m, const float *ids_host, size_t s, lumen_kv_cache **caches, size_t n_caches,
                               const lumen_sample_params *sp, int32_t *token_out) {
    return m ? m->forward_sample(ids_host, s, caches, n_caches, sp, token_out) : LUMEN_ERR_INVALID;
}

size_t lumen_model_weight_bytes(const lumen_model *m) { return m ? m->weight_bytes() : 0; }

int lumen_model_free(lumen_model *m) {
    if (!m) return LUMEN_ERR_INVALID;
    cudaStreamSynchronize(m->ctx->stream);
    m->drop_graphs();
    delete m;
    return LUMEN_OK;
}

}  // extern "C"
