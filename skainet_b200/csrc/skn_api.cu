// C ABI of libskainet_cuda.so: host-pointer / device-pointer front ends of the quantized products.  No exception
// leaves this file.
#include "skn_dense.cuh"

extern "C" {

int32_t skn_dequantize_dev(skn_ctx *ctx, const skn_tensor *t, float *out_dev) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!skn_tensor_ok(t) || t->ctx != ctx) return skn_fail(ctx, SKN_ERR_BAD_HANDLE, "bad tensor handle");
    if (!out_dev) return skn_fail(ctx, SKN_ERR_ARG, "out is NULL");
    if (t->type == SKN_TYPE_BF16) return skn_fail(ctx, SKN_ERR_TYPE, "a dense weight where a block-quantized one is expected");
    if (((uintptr_t)out_dev) & 15) return skn_fail(ctx, SKN_ERR_ALIGN, "output must be 16-byte aligned");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    SKN_CUDA(ctx, skn_launch_dequant(t->type, t->d_blocks, t->pitch, t->n_rows, t->n_cols, out_dev, ctx->stream));
    return SKN_OK;
}

int32_t skn_dequantize(skn_ctx *ctx, const skn_tensor *t, float *out_host) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!skn_tensor_ok(t) || t->ctx != ctx) return skn_fail(ctx, SKN_ERR_BAD_HANDLE, "bad tensor handle");
    if (!out_host) return skn_fail(ctx, SKN_ERR_ARG, "out is NULL");
    const size_t bytes = (size_t)t->n_rows * (size_t)t->n_cols * sizeof(float);
    if (bytes == 0) return SKN_OK;
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    int32_t rc = skn_stage_reserve(ctx, &ctx->d_stage_out, &ctx->d_stage_out_bytes, bytes);
    if (rc) return rc;
    rc = skn_dequantize_dev(ctx, t, (float *)ctx->d_stage_out);
    if (rc) return rc;
    SKN_CUDA(ctx, cudaMemcpyAsync(out_host, ctx->d_stage_out, bytes, cudaMemcpyDeviceToHost, ctx->stream));
    return skn_sync(ctx);
}

static int32_t check_matmul_args(skn_ctx *ctx, const skn_tensor *w, const void *x, int32_t M, int64_t K, const void *y) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    if (!skn_tensor_ok(w) || w->ctx != ctx) return skn_fail(ctx, SKN_ERR_BAD_HANDLE, "bad tensor handle");
    if (M < 0) return skn_fail(ctx, SKN_ERR_ARG, "M is negative");
    if (K != w->n_cols) return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    if (M > 0 && (!x || !y)) return skn_fail(ctx, SKN_ERR_ARG, "x or y is NULL");
    return SKN_OK;
}

}  // extern "C"

// out[m][n] += bias[n]
__global__ void skn_bias_rows_kernel(float *out, const float *bias, int64_t n_rows, int64_t total) {
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) out[i] += bias[i % n_rows];
}

// products with a dense bf16 weight: bf16 rows on the tensor cores from the prefill threshold on, fp32 below
static int32_t dense_matmul(skn_ctx *ctx, const skn_tensor *w, const float *x, int32_t M, const float *bias, float *y) {
    const int64_t K = w->n_cols, ld = (K + 7) / 8 * 8;
    skn_linear l = {};
    l.w = w;
    l.M = M;
    l.x32 = x;
    l.ld_x32 = K;
    l.epi.y32 = y;
    l.epi.ld_y32 = w->n_rows;
    if (ctx->prefill_min_m > 0 && M >= ctx->prefill_min_m) {
        const size_t xb = ((size_t)M * ld * 2 + 255) / 256 * 256, need = xb + SKN_DENSE_MAX_TILES * 4 + SKN_DENSE_WS_FLOATS * 4;
        int32_t rc = skn_stage_reserve(ctx, &ctx->d_scratch, &ctx->d_scratch_bytes, need);
        if (rc) return rc;
        uint8_t *base = (uint8_t *)ctx->d_scratch;
        skn_dense_ws ws = {(float *)(base + xb + SKN_DENSE_MAX_TILES * 4), (unsigned *)(base + xb)};
        SKN_CUDA(ctx, cudaMemsetAsync(ws.tickets, 0, SKN_DENSE_MAX_TILES * 4, ctx->stream));
        SKN_CUDA(ctx, skn_launch_rows_to_bf16(x, K, M, (int)K, (__nv_bfloat16 *)base, ld, ctx->stream));
        l.x16 = (const __nv_bfloat16 *)base;
        l.ld_x16 = ld;
        SKN_CUDA(ctx, skn_launch_dense_tc(ctx, l, ws, ctx->stream));
    } else {
        cudaError_t e = M <= SKN_MATVEC_ROWS ? skn_launch_dense_matvec(ctx, l, ctx->stream) : cudaErrorNotSupported;
        if (e == cudaErrorNotSupported) e = skn_launch_dense_f32(ctx, l, ctx->stream);
        SKN_CUDA(ctx, e);
    }
    if (bias) {
        const int64_t total = (int64_t)M * w->n_rows;
        const int64_t blocks = (total + 255) / 256;
        skn_bias_rows_kernel<<<(unsigned)(blocks < 1184 ? blocks : 1184), 256, 0, ctx->stream>>>(y, bias, w->n_rows, total);
        SKN_CUDA(ctx, cudaGetLastError());
    }
    return SKN_OK;
}

extern "C" {

int32_t skn_matmul_dev(skn_ctx *ctx, const skn_tensor *w, const float *x_dev, int32_t M, int64_t K,
                       const float *bias_dev, float *y_dev) {
    int32_t rc = check_matmul_args(ctx, w, x_dev, M, K, y_dev);
    if (rc) return rc;
    SKN_ENTER(ctx);
    if (M == 0 || w->n_rows == 0) return SKN_OK;
    if ((((uintptr_t)x_dev) & 15) || (((uintptr_t)y_dev) & 15))
        return skn_fail(ctx, SKN_ERR_ALIGN, "x and y must be 16-byte aligned device pointers");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    if (K == 0) {
        // empty reduction: y = bias (or 0)
        SKN_CUDA(ctx, cudaMemsetAsync(y_dev, 0, (size_t)M * w->n_rows * sizeof(float), ctx->stream));
        if (bias_dev)
            for (int32_t m = 0; m < M; ++m)
                SKN_CUDA(ctx, cudaMemcpyAsync(y_dev + (size_t)m * w->n_rows, bias_dev, w->n_rows * sizeof(float),
                                              cudaMemcpyDeviceToDevice, ctx->stream));
        return SKN_OK;
    }
    if (w->type == SKN_TYPE_BF16) return dense_matmul(ctx, w, x_dev, M, bias_dev, y_dev);
    if (ctx->prefill_min_m > 0 && M >= ctx->prefill_min_m && skn_tc_supported(w, M)) {
        // prefill: bf16 copy of the activations, tensor-core matmul with fp32 accumulation
        const size_t ab = (size_t)M * (size_t)K * 2;
        int32_t rc2 = skn_stage_reserve(ctx, &ctx->d_scratch, &ctx->d_scratch_bytes, ab);
        if (rc2) return rc2;
        SKN_CUDA(ctx, skn_launch_f32_to_bf16(x_dev, ctx->d_scratch, (int64_t)M * K, ctx->sm_count, ctx->stream));
        SKN_CUDA(ctx, skn_launch_matmul_tc(ctx, w, ctx->d_scratch, M, bias_dev, y_dev, ctx->stream));
        return SKN_OK;
    }
    SKN_CUDA(ctx, skn_launch_matvec(ctx, w, x_dev, M, bias_dev, y_dev, ctx->stream));
    return SKN_OK;
}

// y[t] = W[t] . x (+ add[t]) for up to three weights that share the activation vector x
int32_t skn_matvec_group_dev(skn_ctx *ctx, int32_t n, const skn_tensor *const *w, const float *x_dev,
                             float *const *y_dev, const float *const *add_dev) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (n < 1 || n > 3 || !w || !y_dev || !x_dev) return skn_fail(ctx, SKN_ERR_ARG, "1 to 3 tensors, non-NULL arrays");
    for (int32_t t = 0; t < n; ++t) {
        if (!skn_tensor_ok(w[t]) || w[t]->ctx != ctx) return skn_fail(ctx, SKN_ERR_BAD_HANDLE, "bad tensor handle");
        if (w[t]->type == SKN_TYPE_BF16) return skn_fail(ctx, SKN_ERR_TYPE, "a dense weight where a block-quantized one is expected");
        if (w[t]->n_cols != w[0]->n_cols) return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
        if (!y_dev[t] || (((uintptr_t)y_dev[t]) & 15)) return skn_fail(ctx, SKN_ERR_ALIGN, "outputs must be 16-byte aligned");
    }
    if (((uintptr_t)x_dev) & 15) return skn_fail(ctx, SKN_ERR_ALIGN, "x must be 16-byte aligned");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    SKN_CUDA(ctx, skn_launch_matvec_group(ctx, n, w, x_dev, y_dev, add_dev, ctx->stream));
    return SKN_OK;
}

int32_t skn_matvec_fused_dev(skn_ctx *ctx, int32_t n, const skn_tensor *const *w, const float *x_dev,
                             float *const *y_dev, const float *const *add_dev, const float *norm_gain_dev,
                             float norm_eps, const float *silu_u_dev) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (n < 1 || n > 3 || !w || !y_dev || !x_dev) return skn_fail(ctx, SKN_ERR_ARG, "1 to 3 tensors, non-NULL arrays");
    if (norm_gain_dev && silu_u_dev) return skn_fail(ctx, SKN_ERR_ARG, "either a norm gain or a SwiGLU partner, not both");
    for (int32_t t = 0; t < n; ++t) {
        if (!skn_tensor_ok(w[t]) || w[t]->ctx != ctx) return skn_fail(ctx, SKN_ERR_BAD_HANDLE, "bad tensor handle");
        if (w[t]->type == SKN_TYPE_BF16) return skn_fail(ctx, SKN_ERR_TYPE, "a dense weight where a block-quantized one is expected");
        if (w[t]->n_cols != w[0]->n_cols) return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
        if (!y_dev[t] || (((uintptr_t)y_dev[t]) & 15)) return skn_fail(ctx, SKN_ERR_ALIGN, "outputs must be 16-byte aligned");
    }
    if ((((uintptr_t)x_dev) | ((uintptr_t)norm_gain_dev) | ((uintptr_t)silu_u_dev)) & 15)
        return skn_fail(ctx, SKN_ERR_ALIGN, "x, gain and partner must be 16-byte aligned");
    const int64_t K = w[0]->n_cols;
    if (K % 4) return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    cudaError_t e = skn_launch_matvec_fused(ctx, n, w, x_dev, y_dev, add_dev, norm_gain_dev, norm_eps, silu_u_dev, ctx->stream);
    if (e == cudaErrorNotSupported) {
        // shapes outside the streaming kernel: transform x with the element-wise kernels first
        const float *xin = x_dev;
        if (norm_gain_dev || silu_u_dev) {
            int32_t rc = skn_stage_reserve(ctx, &ctx->d_scratch, &ctx->d_scratch_bytes, (size_t)K * sizeof(float));
            if (rc) return rc;
            float *t = (float *)ctx->d_scratch;
            if (norm_gain_dev) SKN_CUDA(ctx, skn_launch_rmsnorm(x_dev, norm_gain_dev, t, 1, (int)K, norm_eps, ctx->stream));
            else SKN_CUDA(ctx, skn_launch_silu_mul(x_dev, silu_u_dev, t, K, ctx->sm_count, ctx->stream));
            xin = t;
        }
        e = skn_launch_matvec_group(ctx, n, w, xin, y_dev, add_dev, ctx->stream);
    }
    SKN_CUDA(ctx, e);
    return SKN_OK;
}

int32_t skn_ffn_swiglu_dev(skn_ctx *ctx, const skn_tensor *wg, const skn_tensor *wu, const skn_tensor *wd,
                           const float *x_dev, int32_t M, float *y_dev) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!skn_tensor_ok(wg) || !skn_tensor_ok(wu) || !skn_tensor_ok(wd) || wg->ctx != ctx || wu->ctx != ctx || wd->ctx != ctx)
        return skn_fail(ctx, SKN_ERR_BAD_HANDLE, "bad tensor handle");
    if (M < 0) return skn_fail(ctx, SKN_ERR_ARG, "M is negative");
    if (wg->type == SKN_TYPE_BF16 || wu->type == SKN_TYPE_BF16 || wd->type == SKN_TYPE_BF16) return skn_fail(ctx, SKN_ERR_TYPE, "a dense weight where a block-quantized one is expected");
    if (wg->n_rows != wu->n_rows || wg->n_cols != wu->n_cols || wd->n_cols != wg->n_rows || wg->type != wu->type)
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    if (M == 0 || wd->n_rows == 0) return SKN_OK;
    if (!x_dev || !y_dev) return skn_fail(ctx, SKN_ERR_ARG, "x or y is NULL");
    if ((((uintptr_t)x_dev) | ((uintptr_t)y_dev)) & 15) return skn_fail(ctx, SKN_ERR_ALIGN, "x and y must be 16-byte aligned");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    const int64_t F = wg->n_rows, K = wg->n_cols;
    if (ctx->prefill_min_m > 0 && M >= ctx->prefill_min_m && skn_tc_supported(wg, M) && skn_tc_supported(wd, M)) {
        // [A bf16 | H bf16] in the context scratch
        const size_t ab = ((size_t)M * K * 2 + 255) / 256 * 256, hb = (size_t)M * F * 2;
        int32_t rc = skn_stage_reserve(ctx, &ctx->d_scratch, &ctx->d_scratch_bytes, ab + hb);
        if (rc) return rc;
        void *a16 = ctx->d_scratch, *h16 = (uint8_t *)ctx->d_scratch + ab;
        SKN_CUDA(ctx, skn_launch_f32_to_bf16(x_dev, a16, (int64_t)M * K, ctx->sm_count, ctx->stream));
        SKN_CUDA(ctx, skn_launch_gate_up_tc(ctx, wg, wu, a16, M, h16, ctx->stream));
        SKN_CUDA(ctx, skn_launch_matmul_tc(ctx, wd, h16, M, nullptr, y_dev, ctx->stream));
        return SKN_OK;
    }
    // decode-size path: three fp32 fused dequant-dot products and an element-wise SwiGLU
    const size_t gb = ((size_t)M * F * sizeof(float) + 255) / 256 * 256;
    int32_t rc = skn_stage_reserve(ctx, &ctx->d_scratch, &ctx->d_scratch_bytes, 2 * gb);
    if (rc) return rc;
    float *g = (float *)ctx->d_scratch, *u = (float *)((uint8_t *)ctx->d_scratch + gb);
    SKN_CUDA(ctx, skn_launch_matvec(ctx, wg, x_dev, M, nullptr, g, ctx->stream));
    SKN_CUDA(ctx, skn_launch_matvec(ctx, wu, x_dev, M, nullptr, u, ctx->stream));
    SKN_CUDA(ctx, skn_launch_silu_mul(g, u, g, (int64_t)M * F, ctx->sm_count, ctx->stream));
    SKN_CUDA(ctx, skn_launch_matvec(ctx, wd, g, M, nullptr, y_dev, ctx->stream));
    return SKN_OK;
}

int32_t skn_ffn_swiglu(skn_ctx *ctx, const skn_tensor *wg, const skn_tensor *wu, const skn_tensor *wd,
                       const float *x_host, int32_t M, float *y_host) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!skn_tensor_ok(wg) || !skn_tensor_ok(wd)) return skn_fail(ctx, SKN_ERR_BAD_HANDLE, "bad tensor handle");
    if (M < 0) return skn_fail(ctx, SKN_ERR_ARG, "M is negative");
    if (M == 0) return SKN_OK;
    if (!x_host || !y_host) return skn_fail(ctx, SKN_ERR_ARG, "x or y is NULL");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    const size_t xb = (size_t)M * wg->n_cols * sizeof(float), yb = (size_t)M * wd->n_rows * sizeof(float);
    int32_t rc = skn_stage_reserve(ctx, &ctx->d_stage_in, &ctx->d_stage_in_bytes, xb);
    if (rc) return rc;
    rc = skn_stage_reserve(ctx, &ctx->d_stage_out, &ctx->d_stage_out_bytes, yb);
    if (rc) return rc;
    SKN_CUDA(ctx, cudaMemcpyAsync(ctx->d_stage_in, x_host, xb, cudaMemcpyHostToDevice, ctx->stream));
    rc = skn_ffn_swiglu_dev(ctx, wg, wu, wd, (const float *)ctx->d_stage_in, M, (float *)ctx->d_stage_out);
    if (rc) return rc;
    SKN_CUDA(ctx, cudaMemcpyAsync(y_host, ctx->d_stage_out, yb, cudaMemcpyDeviceToHost, ctx->stream));
    return skn_sync(ctx);
}

// device-side address of a page-locked host buffer (registered or allocated by the CUDA runtime), or NULL for
// pageable memory
static void *host_mapped(const void *p) {
    cudaPointerAttributes a;
    if (cudaPointerGetAttributes(&a, p) != cudaSuccess) {
        cudaGetLastError();
        return nullptr;
    }
    return a.type == cudaMemoryTypeHost ? a.devicePointer : nullptr;
}

// sync: return when y_host holds the result (and report the device status); otherwise return once the
// copies and the launch are enqueued on the context's stream
static int32_t matmul_host(skn_ctx *ctx, const skn_tensor *w, const float *x_host, int32_t M, int64_t K, const float *bias_host,
                           float *y_host, bool sync) {
    int32_t rc = check_matmul_args(ctx, w, x_host, M, K, y_host);
    if (rc) return rc;
    SKN_ENTER(ctx);
    if (M == 0 || w->n_rows == 0) return SKN_OK;
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    // The product reads what the fetch kernel (or the staged copy) of this very call wrote: that chain keeps
    // stream order whatever SKN_OPT_RELAXED_ORDER says about the caller's consecutive calls.
    skn_order_guard guard(ctx);
    const size_t xb = (size_t)M * (size_t)K * sizeof(float);
    const size_t bb = bias_host ? (size_t)w->n_rows * sizeof(float) : 0;
    const size_t xb_al = (xb + 255) / 256 * 256;
    const size_t yb = (size_t)M * (size_t)w->n_rows * sizeof(float);
    rc = skn_stage_reserve(ctx, &ctx->d_stage_in, &ctx->d_stage_in_bytes, xb_al + bb + 256);
    if (rc) return rc;
    float *dx = (float *)ctx->d_stage_in;
    float *db = bias_host ? (float *)((uint8_t *)ctx->d_stage_in + xb_al) : nullptr;
    if (yb <= (64 << 10) && xb <= (1 << 20) && (K % 4) == 0 && ((w->n_rows * (int64_t)M) % 4) == 0 && (!sync || ctx->h_status_dev)) {
        // Decode-size call on page-locked buffers: no copy-engine operation at all.  A one-CTA-per-4-KB kernel
        // fetches x over PCIe into device memory (every CTA of the matvec reads all of x: that must not cross
        // the bus 148 times), and the matvec writes y straight into the caller's mapped buffer.  A copy-engine
        // operation between two kernels costs several microseconds of hand-over each way; kernels hand over
        // to one another in one or two, and the matvec prefetches its weights under the fetch.
        void *xm = host_mapped(x_host), *ym = host_mapped(y_host), *bm = bias_host ? host_mapped(bias_host) : nullptr;
        if (xm && ym && (!bias_host || bm) && !((((uintptr_t)xm) | ((uintptr_t)ym) | ((uintptr_t)bm)) & 15)) {
            SKN_CUDA(ctx, skn_launch_fetch((const float *)xm, dx, (int64_t)M * K, ctx->stream));
            if (db) SKN_CUDA(ctx, skn_launch_fetch((const float *)bm, db, w->n_rows, ctx->stream));
            // (measured: 12.8 us per 4096 x 4096 call this way, 14.8 with a second kernel pushing y out of device
            // memory, 20.2 with a copy-engine transfer of y)
            rc = skn_matmul_dev(ctx, w, dx, M, K, db, (float *)ym);
            if (rc || !sync) return rc;
            // the blocking call: the status word follows through a kernel as well (16 bytes into the pinned mirror)
            SKN_CUDA(ctx, skn_launch_fetch((const float *)ctx->d_status, (float *)ctx->h_status_dev, 4, ctx->stream));
            SKN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
            return skn_status_check(ctx);
        }
    }
    if (sync && yb <= SKN_SMALL_OUT_BYTES) {
        // decode-size result: it is written right below the status word and comes back with it in ONE copy
        // (a separate copy of the status costs as much as the matvec itself)
        const size_t yb_al = (yb + 255) / 256 * 256;
        float *dys = reinterpret_cast<float *>(reinterpret_cast<uint8_t *>(ctx->d_status) - yb_al);
        uint8_t *hys = reinterpret_cast<uint8_t *>(ctx->h_status) - yb_al;
        if (xb) SKN_CUDA(ctx, cudaMemcpyAsync(dx, x_host, xb, cudaMemcpyHostToDevice, ctx->stream));
        if (db) SKN_CUDA(ctx, cudaMemcpyAsync(db, bias_host, bb, cudaMemcpyHostToDevice, ctx->stream));
        rc = skn_matmul_dev(ctx, w, dx, M, K, db, dys);
        if (rc) return rc;
        SKN_CUDA(ctx, cudaMemcpyAsync(hys, dys, yb_al + sizeof(int32_t), cudaMemcpyDeviceToHost, ctx->stream));
        SKN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
        rc = skn_status_check(ctx);
        if (rc) return rc;
        memcpy(y_host, hys, yb);
        return SKN_OK;
    }
    rc = skn_stage_reserve(ctx, &ctx->d_stage_out, &ctx->d_stage_out_bytes, yb);
    if (rc) return rc;
    if (xb) SKN_CUDA(ctx, cudaMemcpyAsync(dx, x_host, xb, cudaMemcpyHostToDevice, ctx->stream));
    if (db) SKN_CUDA(ctx, cudaMemcpyAsync(db, bias_host, bb, cudaMemcpyHostToDevice, ctx->stream));
    rc = skn_matmul_dev(ctx, w, dx, M, K, db, (float *)ctx->d_stage_out);
    if (rc) return rc;
    SKN_CUDA(ctx, cudaMemcpyAsync(y_host, ctx->d_stage_out, yb, cudaMemcpyDeviceToHost, ctx->stream));
    return sync ? skn_sync(ctx) : SKN_OK;
}

int32_t skn_matmul(skn_ctx *ctx, const skn_tensor *w, const float *x_host, int32_t M, int64_t K, const float *bias_host,
                   float *y_host) {
    return matmul_host(ctx, w, x_host, M, K, bias_host, y_host, true);
}

int32_t skn_matmul_async(skn_ctx *ctx, const skn_tensor *w, const float *x_host, int32_t M, int64_t K,
                         const float *bias_host, float *y_host) {
    return matmul_host(ctx, w, x_host, M, K, bias_host, y_host, false);
}

}  // extern "C"

#ifdef SKN_TUNING
// Profiling builds only (never in the shipped library): copies the raw status/trace area.
extern "C" int32_t skn_debug_read_status(skn_ctx *ctx, void *out_host, int64_t bytes) {
    if (!skn_ctx_ok(ctx) || bytes > 32768) return SKN_ERR_ARG;
    SKN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    SKN_CUDA(ctx, cudaMemcpy(out_host, ctx->d_status, (size_t)bytes, cudaMemcpyDeviceToHost));
    return SKN_OK;
}
#endif
