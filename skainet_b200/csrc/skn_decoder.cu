// The shared part of the decoders over dense weights (see skn_decoder.cuh).
#include "skn_decoder.cuh"

constexpr int BF16_MATVEC_ROWS = 2;     // with bf16 operands the tensor-core kernel is faster beyond this

bool skn_decoder::f32() const { return dtype == SKN_DECODER_F32; }
bool skn_decoder::few(int rows) const { return matvec_ok && rows <= (f32() ? SKN_MATVEC_ROWS : BF16_MATVEC_ROWS); }

int skn_decoder::find_rot(double base, int dims) {
    if (dims == 0) return -1;
    for (size_t i = 0; i < rots.size(); ++i)
        if (rots[i].base == base && rots[i].dims == dims) return (int)i;
    rots.push_back(skn_rot_entry{base, dims, nullptr, nullptr});
    return (int)rots.size() - 1;
}

cudaError_t skn_decoder::step_angles(const skn_step &st) {
    cudaError_t e = cudaSuccess;
    for (auto &r : rots)
        if (e == cudaSuccess) e = skn_launch_rot_table(st, r.freq, r.dims / 2, r.table, r.dims / 2, ctx->stream);
    return e;
}

cudaError_t skn_decoder::launch_linear(bool few_rows, const skn_linear &l) {
    if (few_rows) return skn_launch_dense_matvec(ctx, l, ctx->stream);
    if (f32()) return skn_launch_dense_f32(ctx, l, ctx->stream);
    return skn_launch_dense_tc(ctx, l, ws, ctx->stream);
}

cudaError_t skn_decoder::linear(bool few_rows, const skn_tensor *w, int M, const float *in32, int64_t ld32, const __nv_bfloat16 *in16, int64_t ld16,
                                const float *gain, const skn_epi &epi) {
    skn_linear l = {};
    l.w = w;
    l.M = M;
    l.epi = epi;
    l.x32 = in32;
    l.ld_x32 = ld32;
    l.x16 = in16;
    l.ld_x16 = ld16;
    l.gain = gain;
    l.eps = eps;
    return launch_linear(few_rows, l);
}

int32_t skn_decoder::record_layer(int M) {
    const size_t at = trace.size();
    trace.resize(at + (size_t)M * width);
    SKN_CUDA(ctx, cudaMemcpy2DAsync(trace.data() + at, (size_t)width * 4, x, (size_t)ldw * 4, (size_t)width * 4, M, cudaMemcpyDeviceToHost, ctx->stream));
    SKN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    return SKN_OK;
}

int32_t skn_decoder::head(int n, const int32_t *rows) {
    const bool few_rows = few(n);
    const bool fold = few_rows && !rows;
    if (!fold)
        SKN_CUDA(ctx, skn_launch_norm_rows(x, ldw, n, width, eps, nullptr, 0, nullptr, final_norm, h_rows(few_rows || f32()), nullptr, 0, rows, ctx->stream));
    SKN_CUDA(ctx, linear(few_rows, embed, n, fold ? x : h32, ldw, h16, ldw, fold ? final_norm : nullptr,
                         skn_to_rows(SKN_EPI_STORE, logits, vocab, nullptr, 0)));
    return SKN_OK;
}

skn_epi skn_to_rows(int kind, float *y32, int64_t ld32, __nv_bfloat16 *y16, int64_t ld16) {
    skn_epi e = {};
    e.kind = kind;
    e.alpha = 1.f;
    e.y32 = y32; e.ld_y32 = ld32;
    e.y16 = y16; e.ld_y16 = ld16;
    return e;
}

bool skn_dense_is(const skn_tensor *t, const skn_ctx *ctx, int64_t rows, int64_t cols) {
    return skn_tensor_ok(t) && t->ctx == ctx && t->type == SKN_TYPE_BF16 && t->n_rows == rows && t->n_cols == cols;
}

int32_t skn_put_floats(skn_ctx *ctx, float *dst, const float *host, size_t n) {
    SKN_CUDA(ctx, cudaMemcpyAsync(dst, host, sizeof(float) * n, cudaMemcpyHostToDevice, ctx->stream));
    SKN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    return SKN_OK;
}

int32_t skn_decoder_check(skn_ctx *ctx, const skn_decoder_sizes &s) {
    if (s.dtype != SKN_DECODER_F32 && s.dtype != SKN_DECODER_BF16) return skn_fail(ctx, SKN_ERR_TYPE, "unknown decoder number format %d", s.dtype);
    if (s.max_seqs < 1 || s.max_tokens < s.max_seqs || s.max_ctx < 1)
        return skn_fail(ctx, SKN_ERR_ARG, "max_tokens must hold one token of each of max_seqs sequences");
    if (s.n_layers < 1 || s.width < 1 || s.vocab < 1) return skn_fail(ctx, SKN_ERR_ARG, "invalid model geometry");
    if (s.loop_times < 0 || (s.loop_times > 0 && (s.loop_start < 0 || s.loop_stop <= s.loop_start || s.loop_stop > s.n_layers)))
        return skn_fail(ctx, SKN_ERR_ARG, "the loop lies outside the layers");
    return SKN_OK;
}

void skn_decoder_init(skn_decoder *m, int kind, skn_ctx *ctx, const skn_decoder_sizes &s) {
    m->magic = SKN_MAGIC_DECODER;
    m->kind = kind;
    m->ctx = ctx;
    m->max_seqs = s.max_seqs; m->max_tokens = s.max_tokens; m->max_ctx = s.max_ctx; m->dtype = s.dtype; m->n_layers = s.n_layers;
    m->width = s.width; m->vocab = s.vocab; m->eps = s.eps;
    m->embed = nullptr;
    m->matvec_ok = true;
    m->tracing = false;
    m->trace_rows = 0;
    m->ldw = skn_up8(s.width);
    const int a = s.loop_times ? s.loop_start : 0, b = s.loop_times ? s.loop_stop : 0;
    for (int i = 0; i < a; ++i) { m->runs.push_back(i); m->pass.push_back(-1); }
    for (int t = 0; t < s.loop_times; ++t)
        for (int i = a; i < b; ++i) { m->runs.push_back(i); m->pass.push_back(i == a ? t : -1); }
    for (int i = b; i < s.n_layers; ++i) { m->runs.push_back(i); m->pass.push_back(-1); }
    m->host_pos.assign(s.max_seqs, 0);
}

cudaError_t skn_decoder_allocate(skn_decoder *m) {
    const size_t R = m->max_tokens, few = R < SKN_MATVEC_ROWS ? R : SKN_MATVEC_ROWS, r32 = m->f32() ? R : few;
    cudaError_t e = cudaSuccess;
#define DEC_TAKE(p, n) if (e == cudaSuccess) e = m->take(&m->p, n)
    DEC_TAKE(h32, (r32 > SKN_HEAD_ROWS ? r32 : SKN_HEAD_ROWS) * m->ldw);
    DEC_TAKE(h16, m->f32() ? 0 : (R > SKN_HEAD_ROWS ? R : SKN_HEAD_ROWS) * m->ldw);
    DEC_TAKE(logits, (size_t)SKN_HEAD_ROWS * m->vocab);
    DEC_TAKE(ws.partial, m->f32() ? 0 : SKN_DENSE_WS_FLOATS); DEC_TAKE(ws.tickets, m->f32() ? 0 : SKN_DENSE_MAX_TILES);
    DEC_TAKE(final_norm, m->width);
    DEC_TAKE(pos, m->max_seqs); DEC_TAKE(ids_in, R); DEC_TAKE(ids_out, m->max_seqs);
    DEC_TAKE(want, R > (size_t)SKN_HEAD_ROWS ? R : SKN_HEAD_ROWS);
#undef DEC_TAKE
    uint8_t *am = nullptr;
    if (e == cudaSuccess) e = m->take(&am, skn_argmax_scratch_bytes(SKN_HEAD_ROWS));
    m->argmax_scratch = am;
    for (auto &r : m->rots) {
        if (e == cudaSuccess) e = m->take(&r.freq, r.dims / 2);
        if (e == cudaSuccess) e = m->take(&r.table, R * (r.dims / 2));
        if (e == cudaSuccess) {
            std::vector<double> f(r.dims / 2);
            skn_rot_freqs(r.base, r.dims, f.data());
            e = cudaMemcpyAsync(r.freq, f.data(), f.size() * sizeof(double), cudaMemcpyHostToDevice, m->ctx->stream);
            if (e == cudaSuccess) e = cudaStreamSynchronize(m->ctx->stream);
        }
    }
    return e;
}

// the last row of every sequence of the step
__global__ void skn_last_rows_kernel(int32_t *rows, int n, int T) {
    for (int i = threadIdx.x; i < n; i += blockDim.x) rows[i] = i * T + T - 1;
}

extern "C" {

int32_t skn_decoder_destroy(skn_decoder *m) {
    if (!m || m->magic != SKN_MAGIC_DECODER) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    if (skn_ctx_ok(m->ctx)) {
        cudaSetDevice(m->ctx->device);
        cudaStreamSynchronize(m->ctx->stream);
    }
    for (void *p : m->owned) cudaFree(p);
    for (skn_kvcache *k : m->caches) skn_kv_destroy(k);
    for (skn_state *s : m->states) skn_state_destroy(s);
    m->magic = 0;
    delete m;
    return SKN_OK;
}

int32_t skn_decoder_reset(skn_decoder *m, int32_t seq) {
    if (!skn_decoder_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    if (seq < -1 || seq >= m->max_seqs) return skn_fail(ctx, SKN_ERR_ARG, "sequence %d outside [0, %d)", seq, m->max_seqs);
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    // a sequence at position 0 sees no cached key and starts from a zero state: nothing else to clear
    const int a = seq < 0 ? 0 : seq, n = seq < 0 ? m->max_seqs : 1;
    SKN_CUDA(ctx, cudaMemsetAsync(m->pos + a, 0, sizeof(int32_t) * n, ctx->stream));
    for (int i = a; i < a + n; ++i) m->host_pos[i] = 0;
    return SKN_OK;
}

int32_t skn_decoder_position(const skn_decoder *m, int32_t seq) {
    return skn_decoder_ok(m) && seq >= 0 && seq < m->max_seqs ? m->host_pos[seq] : -1;
}

static int32_t check_forward(skn_decoder *m, int32_t seq0, int32_t n_seqs, bool tokens, int32_t T) {
    skn_ctx *ctx = m->ctx;
    if (seq0 < 0 || n_seqs < 1 || n_seqs > SKN_HEAD_ROWS || seq0 + n_seqs > m->max_seqs) return skn_fail(ctx, SKN_ERR_ARG, "sequences outside the decoder");
    if (T < 1 || (int64_t)n_seqs * T > m->max_tokens) return skn_fail(ctx, SKN_ERR_SHAPE, "a step holds at most %d tokens", m->max_tokens);
    if (!tokens && T != 1) return skn_fail(ctx, SKN_ERR_ARG, "tokens may be NULL only for single-token steps");
    for (int s = seq0; s < seq0 + n_seqs; ++s)
        if (m->host_pos[s] + T > m->max_ctx) return skn_fail(ctx, SKN_ERR_SHAPE, "context of %d tokens exceeded", m->max_ctx);
    if (!m->embed) return skn_fail(ctx, SKN_ERR_ARG, "model head not set");
    if (!m->ready()) return skn_fail(ctx, SKN_ERR_ARG, "a layer has no weights");
    return SKN_OK;
}

int32_t skn_decoder_forward_dev(skn_decoder *m, int32_t seq0, int32_t n_seqs, const int32_t *tokens_dev, int32_t T, int32_t head) {
    if (!skn_decoder_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    int32_t rc = check_forward(m, seq0, n_seqs, tokens_dev != nullptr, T);
    if (rc) return rc;
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    const skn_step st = {seq0, n_seqs, T, m->pos, m->max_ctx};
    if (m->tracing) {
        m->trace.clear();
        m->trace_rows = n_seqs * T;
    }
    rc = m->run_layers(st, tokens_dev ? tokens_dev : m->ids_out + seq0);
    if (rc == SKN_OK) {
        const cudaError_t e = skn_launch_advance(st, m->pos, ctx->d_status, ctx->stream);
        if (e != cudaSuccess) rc = skn_check_cuda(ctx, e, "advance");
    }
    if (rc == SKN_OK)
        for (int s = seq0; s < seq0 + n_seqs; ++s) m->host_pos[s] += T;
    if (rc == SKN_OK && head) {
        if (T > 1) skn_last_rows_kernel<<<1, 64, 0, ctx->stream>>>(m->want, n_seqs, T);
        rc = m->head(n_seqs, T > 1 ? m->want : nullptr);
        if (rc == SKN_OK) {
            const cudaError_t e = skn_launch_argmax(m->logits, n_seqs, m->vocab, m->ids_out + seq0, m->argmax_scratch, ctx->stream);
            if (e != cudaSuccess) rc = skn_check_cuda(ctx, e, "argmax");
        }
    }
    return rc;
}

int32_t skn_decoder_forward(skn_decoder *m, int32_t seq0, int32_t n_seqs, const int32_t *tokens_host, int32_t T, int32_t n_want,
                            const int32_t *want_rows_host, float *logits_host, int32_t *next_host) {
    if (!skn_decoder_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    int32_t rc = check_forward(m, seq0, n_seqs, tokens_host != nullptr, T);
    if (rc) return rc;
    if (n_want < 0 || n_want > n_seqs * T || (n_want && (!want_rows_host || !logits_host))) return skn_fail(ctx, SKN_ERR_ARG, "bad list of wanted rows");
    for (int i = 0; i < n_want; ++i)
        if (want_rows_host[i] < 0 || want_rows_host[i] >= n_seqs * T) return skn_fail(ctx, SKN_ERR_ARG, "a wanted row lies outside the step");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    if (tokens_host) SKN_CUDA(ctx, cudaMemcpyAsync(m->ids_in, tokens_host, sizeof(int32_t) * n_seqs * T, cudaMemcpyHostToDevice, ctx->stream));
    rc = skn_decoder_forward_dev(m, seq0, n_seqs, tokens_host ? m->ids_in : nullptr, T, next_host != nullptr);
    if (rc == SKN_OK && next_host)
        SKN_CUDA(ctx, cudaMemcpyAsync(next_host, m->ids_out + seq0, sizeof(int32_t) * n_seqs, cudaMemcpyDeviceToHost, ctx->stream));
    for (int i = 0; i < n_want && rc == SKN_OK; i += SKN_HEAD_ROWS) {
        const int n = n_want - i < SKN_HEAD_ROWS ? n_want - i : SKN_HEAD_ROWS;
        SKN_CUDA(ctx, cudaMemcpyAsync(m->want, want_rows_host + i, sizeof(int32_t) * n, cudaMemcpyHostToDevice, ctx->stream));
        rc = m->head(n, m->want);
        if (rc == SKN_OK)
            SKN_CUDA(ctx, cudaMemcpyAsync(logits_host + (size_t)i * m->vocab, m->logits, sizeof(float) * n * m->vocab, cudaMemcpyDeviceToHost, ctx->stream));
    }
    return rc ? rc : skn_sync(ctx);
}

int32_t skn_decoder_trace(skn_decoder *m, int32_t on, int32_t rows, float *out_host) {
    if (!skn_decoder_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    m->tracing = on != 0;
    if (!out_host) return SKN_OK;
    const size_t n = m->runs.size() * (size_t)rows * m->width;
    if (rows != m->trace_rows || m->trace.size() != n) return skn_fail(ctx, SKN_ERR_ARG, "the last step recorded %d rows", m->trace_rows);
    memcpy(out_host, m->trace.data(), n * sizeof(float));
    return SKN_OK;
}

}  // extern "C"
