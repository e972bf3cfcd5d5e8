// Allocation and description of what a decoder keeps between steps: KV caches (rings that count their own tokens,
// and position-addressed ones whose owner does) and recurrent states.
#include "skn_internal.cuh"

#include <new>

bool skn_kv_ok(const skn_kvcache *kv) { return kv && kv->magic == SKN_MAGIC_KV && skn_ctx_ok(kv->ctx); }

extern "C" {

int32_t skn_kv_create(skn_ctx *ctx, int32_t batch, int32_t n_kv_heads, int32_t head_dim, int32_t capacity,
                      skn_kvcache **out) {
    return skn_kv_create_typed(ctx, batch, n_kv_heads, head_dim, capacity, SKN_KV_F32, out);
}

int32_t skn_kv_create_typed(skn_ctx *ctx, int32_t batch, int32_t n_kv_heads, int32_t head_dim, int32_t capacity,
                            int32_t kv_dtype, skn_kvcache **out) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!out) return skn_fail(ctx, SKN_ERR_ARG, "out is NULL");
    *out = nullptr;
    if (kv_dtype != SKN_KV_F32 && kv_dtype != SKN_KV_F16 && kv_dtype != SKN_KV_Q8_0)
        return skn_fail(ctx, SKN_ERR_TYPE, "cache element type %d is none of fp32, fp16, Q8_0", kv_dtype);
    if (batch < 1 || n_kv_heads < 1 || capacity < 1) return skn_fail(ctx, SKN_ERR_ARG, "batch, heads and capacity must be positive");
    if (head_dim != 64 && head_dim != 128) return skn_fail(ctx, SKN_ERR_SHAPE, "head_dim must be 64 or 128 (got %d)", head_dim);
    skn_kvcache *kv = new (std::nothrow) skn_kvcache();
    if (!kv) return skn_fail(ctx, SKN_ERR_OOM, "host allocation failed");
    memset(kv, 0, sizeof(*kv));
    kv->magic = SKN_MAGIC_KV;
    kv->ctx = ctx;
    kv->batch = batch; kv->n_kv_heads = n_kv_heads; kv->head_dim = head_dim; kv->capacity = capacity;
    kv->dtype = kv_dtype;
    kv->v_dim = kv->k_pitch = kv->v_pitch = kv->v_stride = head_dim;
    // Q8_0: an int8 plane, then the fp16 scales of its 32-dim blocks
    const size_t elems = (size_t)batch * n_kv_heads * capacity * head_dim;
    const size_t n = kv_dtype == SKN_KV_Q8_0 ? elems + elems / 32 * 2 : elems * (kv_dtype == SKN_KV_F16 ? 2 : sizeof(float));
    cudaError_t e = cudaSetDevice(ctx->device);
    if (e == cudaSuccess) e = cudaMalloc((void **)&kv->d_k, n);
    if (e == cudaSuccess) e = cudaMalloc((void **)&kv->d_v, n);
    const size_t n_ints = (size_t)2 * batch + (size_t)batch * n_kv_heads;     // lengths, starts, merge tickets
    if (e == cudaSuccess) e = cudaMalloc((void **)&kv->d_len, n_ints * sizeof(int32_t));
    if (e == cudaSuccess) {
        kv->d_start = kv->d_len + batch;
        kv->d_tickets = reinterpret_cast<unsigned *>(kv->d_len + 2 * batch);
        e = cudaMemsetAsync(kv->d_len, 0, n_ints * sizeof(int32_t), ctx->stream);
    }
    if (e == cudaSuccess) e = cudaStreamSynchronize(ctx->stream);
    if (e != cudaSuccess) {
        if (kv->d_k) cudaFree(kv->d_k);
        if (kv->d_v) cudaFree(kv->d_v);
        if (kv->d_len) cudaFree(kv->d_len);
        kv->magic = 0;
        delete kv;
        return skn_check_cuda(ctx, e, "kv cache allocation");
    }
    *out = kv;
    return SKN_OK;
}

int32_t skn_kv_destroy(skn_kvcache *kv) {
    if (!kv || kv->magic != SKN_MAGIC_KV) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad kv cache handle");
    if (skn_ctx_ok(kv->ctx)) {
        cudaSetDevice(kv->ctx->device);
        cudaStreamSynchronize(kv->ctx->stream);
    }
    cudaFree(kv->d_k);
    cudaFree(kv->d_v);
    cudaFree(kv->d_len);
    kv->magic = 0;
    delete kv;
    return SKN_OK;
}

int32_t skn_kv_reset(skn_kvcache *kv) {
    if (!skn_kv_ok(kv)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad kv cache handle");
    skn_ctx *ctx = kv->ctx;
    SKN_ENTER(ctx);
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    SKN_CUDA(ctx, cudaMemsetAsync(kv->d_len, 0, 2 * sizeof(int32_t) * kv->batch, ctx->stream));
    return SKN_OK;
}

int32_t skn_kv_create_by_position(skn_ctx *ctx, int32_t batch, int32_t n_kv_heads, int32_t k_dim, int32_t v_dim, int32_t capacity,
                                  int32_t kv_dtype, skn_kvcache **out) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!out) return skn_fail(ctx, SKN_ERR_ARG, "out is NULL");
    *out = nullptr;
    if (kv_dtype != SKN_KV_F32 && kv_dtype != SKN_KV_BF16)
        return skn_fail(ctx, SKN_ERR_TYPE, "a position-addressed cache holds fp32 or bf16, not element type %d", kv_dtype);
    if (batch < 1 || n_kv_heads < 1 || capacity < 1 || k_dim < 1 || v_dim < 0)
        return skn_fail(ctx, SKN_ERR_ARG, "batch, heads, widths and capacity must be positive");
    if (k_dim > SKN_KV_MAX_DIM || v_dim > SKN_KV_MAX_DIM)
        return skn_fail(ctx, SKN_ERR_SHAPE, "head widths of %d and %d are above %d", k_dim, v_dim, SKN_KV_MAX_DIM);
    skn_kvcache *kv = new (std::nothrow) skn_kvcache();
    if (!kv) return skn_fail(ctx, SKN_ERR_OOM, "host allocation failed");
    memset(kv, 0, sizeof(*kv));
    kv->magic = SKN_MAGIC_KV;
    kv->ctx = ctx;
    kv->batch = batch; kv->n_kv_heads = n_kv_heads; kv->head_dim = k_dim; kv->v_dim = v_dim; kv->capacity = capacity;
    kv->dtype = kv_dtype;
    kv->by_position = true;
    kv->k_pitch = (k_dim + 15) / 16 * 16;        // whole k-steps of the tensor-core kernel; the padding stays zero
    kv->v_pitch = kv->v_stride = (v_dim + 15) / 16 * 16;
    const size_t es = kv_dtype == SKN_KV_F32 ? 4 : 2, rows = (size_t)batch * n_kv_heads * capacity;
    cudaError_t e = cudaSetDevice(ctx->device);
    if (e == cudaSuccess) e = cudaMalloc(&kv->d_k, rows * kv->k_pitch * es);
    if (e == cudaSuccess && v_dim) e = cudaMalloc(&kv->d_v, rows * kv->v_pitch * es);
    if (e == cudaSuccess) e = cudaMalloc((void **)&kv->d_len, 2 * batch * sizeof(int32_t));
    if (e == cudaSuccess) {
        kv->d_start = kv->d_len + batch;
        e = cudaMemsetAsync(kv->d_len, 0, 2 * batch * sizeof(int32_t), ctx->stream);
    }
    if (e == cudaSuccess) e = cudaMemsetAsync(kv->d_k, 0, rows * kv->k_pitch * es, ctx->stream);
    if (e == cudaSuccess && v_dim) e = cudaMemsetAsync(kv->d_v, 0, rows * kv->v_pitch * es, ctx->stream);
    if (e == cudaSuccess) e = cudaStreamSynchronize(ctx->stream);
    if (e != cudaSuccess) {
        skn_kv_destroy(kv);
        return skn_check_cuda(ctx, e, "kv cache allocation");
    }
    *out = kv;
    return SKN_OK;
}

// element type of the cache buffers (SKN_KV_F32 / SKN_KV_F16 / SKN_KV_Q8_0): what the pointers of skn_kv_info point at
int32_t skn_kv_dtype(const skn_kvcache *kv, int32_t *kv_dtype) {
    if (!skn_kv_ok(kv)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad kv cache handle");
    if (!kv_dtype) return skn_fail(kv->ctx, SKN_ERR_ARG, "kv_dtype is NULL");
    *kv_dtype = kv->dtype;
    return SKN_OK;
}

// device pointers of the cache (for callers that fill it with their own kernels)
int32_t skn_kv_info(const skn_kvcache *kv, int32_t *batch, int32_t *n_kv_heads, int32_t *head_dim, int32_t *capacity,
                    void **k_dev, void **v_dev, void **len_dev, void **start_dev) {
    if (!skn_kv_ok(kv)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad kv cache handle");
    if (batch) *batch = kv->batch;
    if (n_kv_heads) *n_kv_heads = kv->n_kv_heads;
    if (head_dim) *head_dim = kv->head_dim;
    if (capacity) *capacity = kv->capacity;
    if (k_dev) *k_dev = kv->d_k;
    if (v_dev) *v_dev = kv->d_v;
    if (len_dev) *len_dev = kv->d_len;
    if (start_dev) *start_dev = kv->d_start;
    return SKN_OK;
}

int32_t skn_state_create(skn_ctx *ctx, int32_t slots, int32_t heads, int32_t k_dim, int32_t v_dim, skn_state **out) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!out) return skn_fail(ctx, SKN_ERR_ARG, "out is NULL");
    *out = nullptr;
    if (slots < 1 || heads < 1 || k_dim < 1 || v_dim < 1) return skn_fail(ctx, SKN_ERR_ARG, "slots, heads and widths must be positive");
    skn_state *s = new (std::nothrow) skn_state();
    if (!s) return skn_fail(ctx, SKN_ERR_OOM, "host allocation failed");
    s->magic = SKN_MAGIC_STATE;
    s->ctx = ctx;
    s->slots = slots; s->heads = heads; s->k_dim = k_dim; s->v_dim = v_dim;
    s->v_pitch = (v_dim + 3) / 4 * 4;
    s->d = nullptr;
    const size_t bytes = (size_t)slots * heads * k_dim * s->v_pitch * sizeof(float);
    cudaError_t e = cudaSetDevice(ctx->device);
    if (e == cudaSuccess) e = cudaMalloc((void **)&s->d, bytes);
    if (e == cudaSuccess) e = cudaMemsetAsync(s->d, 0, bytes, ctx->stream);
    if (e == cudaSuccess) e = cudaStreamSynchronize(ctx->stream);
    if (e != cudaSuccess) {
        skn_state_destroy(s);
        return skn_check_cuda(ctx, e, "recurrent state allocation");
    }
    *out = s;
    return SKN_OK;
}

int32_t skn_state_destroy(skn_state *s) {
    if (!s || s->magic != SKN_MAGIC_STATE) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad state handle");
    if (skn_ctx_ok(s->ctx)) {
        cudaSetDevice(s->ctx->device);
        cudaStreamSynchronize(s->ctx->stream);
    }
    if (s->d) cudaFree(s->d);
    s->magic = 0;
    delete s;
    return SKN_OK;
}

int32_t skn_state_read(skn_state *s, int32_t slot, float *out_host) {
    if (!s || s->magic != SKN_MAGIC_STATE || !skn_ctx_ok(s->ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad state handle");
    skn_ctx *ctx = s->ctx;
    SKN_ENTER(ctx);
    if (slot < 0 || slot >= s->slots || !out_host) return skn_fail(ctx, SKN_ERR_ARG, "slot out of range or NULL output");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    const size_t rows = (size_t)s->heads * s->k_dim;
    SKN_CUDA(ctx, cudaMemcpy2DAsync(out_host, (size_t)s->v_dim * 4, s->d + (size_t)slot * rows * s->v_pitch, (size_t)s->v_pitch * 4,
                                    (size_t)s->v_dim * 4, rows, cudaMemcpyDeviceToHost, ctx->stream));
    return skn_sync(ctx);
}

}  // extern "C"
