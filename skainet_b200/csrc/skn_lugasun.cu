// The Lugasun decoder over dense bf16 weights: one step is a fixed sequence of launches on the context's stream, all
// with programmatic dependent launch and capturable in a CUDA graph.  Three routes share the buffers and the mixers:
//
//   few rows                        fp32 activations: norm + joint projection | attention + state update | output
//                                   projection + residual | norm + up + relu^2 | down + residual | token side input
//   bf16, more rows                 tcgen05 products of bf16 rows; relu^2, the residual sum and the side gate in their
//                                   epilogues, norms as row kernels (the side input's norm joins the next layer's)
//   fp32, more rows                 the same sequence with fp32 rows and fp32 products
//
// The residual stream, scores, softmax, norms, angles, decays and states are fp32 in every route.
#include "skn_mixers.cuh"
#include "skn_ptx.cuh"

#include <math.h>
#include <new>
#include <stdlib.h>
#include <vector>

#define SKN_MAGIC_LUGASUN 0x736b6e75u   // 'sknu'

namespace {

struct Layer {
    skn_lugasun_layer spec;
    std::vector<double> decay;
    skn_lugasun_weights w;                       // tensors (gains below, on the device)
    float *norm1, *norm2, *q_gain, *k_gain, *side_norm, *powers;
    int rot_l, rot_r;                            // index of the rotation table, -1: none
};

struct Rot {
    double base;
    int dims;
    double *freq;
    float2 *table;
};

constexpr int BF16_MATVEC_ROWS = 2;
constexpr int SIDE_ROWS = 16;                    // rows whose token side input takes one launch
constexpr int HEAD_ROWS = 64;                    // rows of logits computed at a time

inline int64_t up8(int64_t n) { return (n + 7) / 8 * 8; }

}

struct skn_lugasun {
    uint32_t magic;
    skn_ctx *ctx;
    skn_lugasun_spec spec;
    int32_t max_seqs, max_tokens, max_ctx, dtype;
    std::vector<Layer> layers;
    std::vector<int> runs;                       // layer index of every layer run
    std::vector<char> pass_start;                // a pass of the loop begins before this run
    std::vector<skn_kvcache *> kv;               // per run
    std::vector<skn_state *> state;
    std::vector<Rot> rots;
    std::vector<void *> owned;                   // device allocations
    const skn_tensor *embed, *loop_in, *side_embed;
    float *final_norm;
    std::vector<int32_t> host_pos;
    int32_t *pos, *ids_in, *ids_out, *want;
    bool matvec_ok;
    // activations
    int64_t ldw, ldp, ldm, ldf, lds;             // row pitches: width, joint projection, mixer output, feed-forward, side
    float *xa, *xb;                              // the residual stream alternates between two buffers where a pass of the loop starts
    float *x, *xalt;                             // the current one and the other (x: the last step's result between steps)
    float *x0, *proj, *h32, *mix32, *u32, *g32, *y32, *logits;
    __nv_bfloat16 *h16, *mix16, *u16, *g16, *cat16, *x16, *q16;
    float *attn_scratch, *ret_chunks;
    unsigned *tickets;
    skn_dense_ws ws;
    void *argmax_scratch;
    // recording of the residual stream
    bool tracing;
    std::vector<float> trace;
    int trace_rows;
};

static bool lug_ok(const skn_lugasun *m) { return m && m->magic == SKN_MAGIC_LUGASUN && skn_ctx_ok(m->ctx); }

template <class T> static cudaError_t take(skn_lugasun *m, T **p, size_t n) {
    *p = nullptr;
    if (n == 0) return cudaSuccess;
    const cudaError_t e = cudaMalloc((void **)p, n * sizeof(T));
    if (e != cudaSuccess) return e;
    m->owned.push_back(*p);
    return cudaMemsetAsync(*p, 0, n * sizeof(T), m->ctx->stream);      // row padding stays zero
}

static int find_rot(skn_lugasun *m, double base, int dims) {
    if (dims == 0) return -1;
    for (size_t i = 0; i < m->rots.size(); ++i)
        if (m->rots[i].base == base && m->rots[i].dims == dims) return (int)i;
    m->rots.push_back(Rot{base, dims, nullptr, nullptr});
    return (int)m->rots.size() - 1;
}

static int64_t in_rows(const skn_lugasun_layer &l) {
    return (int64_t)l.left.heads * l.left.dim + (int64_t)l.left.kv_heads * (l.left.dim + l.left.vdim) +
           (int64_t)l.right.heads * (2 * l.right.dim + 2 * l.right.vdim);
}
static int64_t out_cols(const skn_lugasun_layer &l) { return (int64_t)l.left.heads * l.left.vdim + (int64_t)l.right.heads * l.right.vdim; }

static int32_t check_spec(skn_ctx *ctx, const skn_lugasun_spec *s) {
    if (s->n_layers < 1 || s->width < 1 || s->vocab < 1 || s->side_dim < 0 || !s->layers) return skn_fail(ctx, SKN_ERR_ARG, "invalid model geometry");
    if (s->loop_times < 0 || (s->loop_times > 0 && (s->loop_start < 0 || s->loop_stop <= s->loop_start || s->loop_stop > s->n_layers)))
        return skn_fail(ctx, SKN_ERR_ARG, "the loop lies outside the layers");
    for (int i = 0; i < s->n_layers; ++i) {
        int32_t rc = skn_check_attn_spec(ctx, &s->layers[i].left);
        if (!rc) rc = skn_check_retention_spec(ctx, &s->layers[i].right);
        if (rc) return rc;
        if (s->layers[i].ff < 0) return skn_fail(ctx, SKN_ERR_ARG, "negative feed-forward width");
    }
    return SKN_OK;
}

static cudaError_t allocate(skn_lugasun *m) {
    const skn_lugasun_spec &s = m->spec;
    const bool f32 = m->dtype == SKN_LUGASUN_F32;
    const size_t R = m->max_tokens, few = R < SKN_MATVEC_ROWS ? R : SKN_MATVEC_ROWS, r32 = f32 ? R : few, r16 = f32 ? 0 : R;
    int64_t P = 0, X = 0, F = 0;
    size_t scratch = 1, tick = 1, chunks = 1, q16 = 0;
    const size_t max_chunks = R / SKN_RET_CHUNK + m->max_seqs + 1;
    for (size_t i = 0; i < m->runs.size(); ++i) {
        const skn_lugasun_layer &l = m->layers[m->runs[i]].spec;
        P = in_rows(l) > P ? in_rows(l) : P;
        X = out_cols(l) > X ? out_cols(l) : X;
        F = l.ff > F ? l.ff : F;
        // rows that meet the split kernel: single-token steps, and every row where the tensor-core form does not apply
        const size_t rows = skn_chunk_attn_tc(m->kv[i]) ? (size_t)m->max_seqs : R;
        const size_t a = skn_chunk_attn_scratch((int)rows, l.left.heads, l.left.vdim, l.left.chunk, m->max_ctx);
        scratch = a > scratch ? a : scratch;
        tick = rows * l.left.heads > tick ? rows * l.left.heads : tick;
        const size_t c = max_chunks * l.right.heads * l.right.dim * m->state[i]->v_pitch;
        chunks = c > chunks ? c : chunks;
        const size_t q = R * l.left.heads * m->kv[i]->k_pitch;
        if (skn_chunk_attn_tc(m->kv[i]) && q > q16) q16 = q;
    }
    m->ldw = up8(s.width); m->ldp = up8(P); m->ldm = up8(X); m->ldf = up8(F); m->lds = up8(s.side_dim);
    const int64_t ldc = up8(2 * (int64_t)s.width);
    cudaError_t e = cudaSuccess;
#define LUG_TAKE(p, n) if (e == cudaSuccess) e = take(m, &m->p, n)
    LUG_TAKE(xa, R * m->ldw); LUG_TAKE(xb, R * m->ldw); LUG_TAKE(x0, R * m->ldw);
    LUG_TAKE(proj, R * m->ldp);
    LUG_TAKE(h32, (r32 > HEAD_ROWS ? r32 : HEAD_ROWS) * m->ldw); LUG_TAKE(mix32, r32 * m->ldm); LUG_TAKE(u32, r32 * m->ldf); LUG_TAKE(g32, r32 * m->lds);
    LUG_TAKE(y32, s.side_dim ? R * m->ldw : 0);
    LUG_TAKE(h16, f32 ? 0 : (R > HEAD_ROWS ? R : HEAD_ROWS) * m->ldw); LUG_TAKE(mix16, r16 * m->ldm); LUG_TAKE(u16, r16 * m->ldf); LUG_TAKE(g16, r16 * m->lds);
    LUG_TAKE(cat16, s.loop_times ? r16 * ldc : 0); LUG_TAKE(x16, s.side_dim ? r16 * m->ldw : 0); LUG_TAKE(q16, q16);
    LUG_TAKE(logits, (size_t)HEAD_ROWS * s.vocab);
    LUG_TAKE(attn_scratch, scratch); LUG_TAKE(tickets, tick); LUG_TAKE(ret_chunks, chunks);
    LUG_TAKE(ws.partial, f32 ? 0 : SKN_DENSE_WS_FLOATS); LUG_TAKE(ws.tickets, f32 ? 0 : SKN_DENSE_MAX_TILES);
    LUG_TAKE(final_norm, s.width);
    LUG_TAKE(pos, m->max_seqs); LUG_TAKE(ids_in, R); LUG_TAKE(ids_out, m->max_seqs); LUG_TAKE(want, R > (size_t)HEAD_ROWS ? R : HEAD_ROWS);
#undef LUG_TAKE
    uint8_t *am = nullptr;
    if (e == cudaSuccess) e = take(m, &am, skn_argmax_scratch_bytes(HEAD_ROWS));
    m->argmax_scratch = am;
    for (auto &l : m->layers) {
        if (e == cudaSuccess) e = take(m, &l.norm1, s.width);
        if (e == cudaSuccess) e = take(m, &l.norm2, s.width);
        if (e == cudaSuccess) e = take(m, &l.side_norm, s.width);
        if (e == cudaSuccess) e = take(m, &l.q_gain, l.spec.left.dim);
        if (e == cudaSuccess) e = take(m, &l.k_gain, l.spec.left.dim);
        const size_t np = (size_t)l.spec.right.heads * (SKN_RET_CHUNK + 1);
        if (e == cudaSuccess) e = take(m, &l.powers, np);
        if (e == cudaSuccess) {
            std::vector<float> pw(np);
            skn_decay_powers(l.decay.data(), l.spec.right.heads, pw.data());
            e = cudaMemcpyAsync(l.powers, pw.data(), np * sizeof(float), cudaMemcpyHostToDevice, m->ctx->stream);
            if (e == cudaSuccess) e = cudaStreamSynchronize(m->ctx->stream);
        }
    }
    for (auto &r : m->rots) {
        if (e == cudaSuccess) e = take(m, &r.freq, r.dims / 2);
        if (e == cudaSuccess) e = take(m, &r.table, R * (r.dims / 2));
        if (e == cudaSuccess) {
            std::vector<double> f(r.dims / 2);
            skn_rot_freqs(r.base, r.dims, f.data());
            e = cudaMemcpyAsync(r.freq, f.data(), f.size() * sizeof(double), cudaMemcpyHostToDevice, m->ctx->stream);
            if (e == cudaSuccess) e = cudaStreamSynchronize(m->ctx->stream);
        }
    }
    return e;
}

static int32_t put_gain(skn_lugasun *m, float *dst, const float *host, int n) {
    SKN_CUDA(m->ctx, cudaMemcpyAsync(dst, host, sizeof(float) * n, cudaMemcpyHostToDevice, m->ctx->stream));
    SKN_CUDA(m->ctx, cudaStreamSynchronize(m->ctx->stream));
    return SKN_OK;
}

static bool dense_is(const skn_tensor *t, const skn_ctx *ctx, int64_t rows, int64_t cols) {
    return skn_tensor_ok(t) && t->ctx == ctx && t->type == SKN_TYPE_BF16 && t->n_rows == rows && t->n_cols == cols;
}

// a weight row and one activation row in the matvec kernel's shared memory
static bool fits_matvec(const skn_tensor *t) { return !t || t->pitch <= 64 * 1024; }

// rows of a step that take the matvec route; with bf16 operands the tensor-core kernel is faster beyond BF16_MATVEC_ROWS
static bool is_few(const skn_lugasun *m, int rows) {
    return m->matvec_ok && rows <= (m->dtype == SKN_LUGASUN_F32 ? SKN_MATVEC_ROWS : BF16_MATVEC_ROWS);
}

// The three routes of a linear layer.  in32 / in16: the same rows in either form (in16 only where bf16 rows run).
static cudaError_t linear(skn_lugasun *m, bool few, const skn_tensor *w, int M, const float *in32, int64_t ld32, const __nv_bfloat16 *in16,
                          int64_t ld16, const float *gain, const skn_epi &epi) {
    skn_linear l = {};
    l.w = w;
    l.M = M;
    l.epi = epi;
    l.x32 = in32;
    l.ld_x32 = ld32;
    l.x16 = in16;
    l.ld_x16 = ld16;
    l.gain = gain;
    l.eps = m->spec.eps;
    if (few) return skn_launch_dense_matvec(m->ctx, l, m->ctx->stream);
    if (m->dtype == SKN_LUGASUN_F32) return skn_launch_dense_f32(m->ctx, l, m->ctx->stream);
    return skn_launch_dense_tc(m->ctx, l, m->ws, m->ctx->stream);
}

static skn_epi to_rows(int kind, float *y32, int64_t ld32, __nv_bfloat16 *y16, int64_t ld16) {
    skn_epi e = {};
    e.kind = kind;
    e.y32 = y32; e.ld_y32 = ld32;
    e.y16 = y16; e.ld_y16 = ld16;
    return e;
}

// the step's layers; leaves the residual stream in m->x
static int32_t run_layers(skn_lugasun *m, const skn_step &st, const int32_t *ids) {
    skn_ctx *ctx = m->ctx;
    cudaStream_t s = ctx->stream;
    const skn_lugasun_spec &sp = m->spec;
    const int M = st.n_seqs * st.T, W = sp.width;
    const bool f32 = m->dtype == SKN_LUGASUN_F32, few = is_few(m, M), rows32 = few || f32;
    const int64_t ldw = m->ldw;
    m->x = m->xa;
    m->xalt = m->xb;
    SKN_CUDA(ctx, skn_launch_embed_bf16(m->embed, ids, M, m->x, sp.loop_times ? m->x0 : nullptr, ldw, s));
    for (auto &r : m->rots) SKN_CUDA(ctx, skn_launch_rot_table(st, r.freq, r.dims / 2, r.table, r.dims / 2, s));
    const skn_rows_out hout = rows32 ? skn_rows_out{m->h32, ldw, nullptr, 0} : skn_rows_out{nullptr, 0, m->h16, ldw};
    bool h_ready = false;                        // the first norm of this run was written by the run before
    for (size_t run = 0; run < m->runs.size(); ++run) {
        Layer &l = m->layers[m->runs[run]];
        if (m->pass_start[run]) {
            // x <- W_in [x; x0]
            skn_linear in = {};
            in.w = m->loop_in;
            in.M = M;
            in.epi = to_rows(SKN_EPI_STORE, m->xalt, ldw, nullptr, 0);
            if (rows32) {
                in.x32 = m->x; in.ld_x32 = ldw; in.x32b = m->x0; in.ld_x32b = ldw; in.k_a = W;
                SKN_CUDA(ctx, few ? skn_launch_dense_matvec(ctx, in, s) : skn_launch_dense_f32(ctx, in, s));
            } else {
                const int64_t ldc = up8(2 * (int64_t)W);
                SKN_CUDA(ctx, skn_launch_concat_bf16(m->x, m->x0, ldw, M, W, m->cat16, ldc, s));
                in.x16 = m->cat16; in.ld_x16 = ldc;
                SKN_CUDA(ctx, skn_launch_dense_tc(ctx, in, m->ws, s));
            }
            float *t = m->x; m->x = m->xalt; m->xalt = t;
            h_ready = false;
        }
        // mixer
        if (!few && !h_ready) SKN_CUDA(ctx, skn_launch_norm_rows(m->x, ldw, M, W, sp.eps, nullptr, 0, nullptr, l.norm1, hout, nullptr, 0, nullptr, s));
        const skn_attn_spec &a = l.spec.left;
        const skn_retention_spec &r = l.spec.right;
        SKN_CUDA(ctx, linear(m, few, l.w.w_in, M, few ? m->x : m->h32, ldw, m->h16, ldw, few ? l.norm1 : nullptr,
                             to_rows(SKN_EPI_STORE, m->proj, m->ldp, nullptr, 0)));
        skn_attn_args aa = {};
        aa.kv = m->kv[run]; aa.heads = a.heads; aa.chunk = a.chunk; aa.scale = a.scale; aa.softcap = a.softcap; aa.eps = sp.eps;
        aa.q_gain = l.q_gain; aa.k_gain = l.k_gain;
        if (l.rot_l >= 0) aa.rot = skn_rot{m->rots[l.rot_l].table, a.rot_dims / 2, a.rot_dims / 2};
        aa.q = m->proj; aa.k = aa.q + (int64_t)a.heads * a.dim; aa.v = aa.k + (int64_t)a.kv_heads * a.dim; aa.ld = m->ldp;
        aa.out_scale = l.spec.left_scale;
        aa.scratch = m->attn_scratch; aa.tickets = m->tickets; aa.q16 = m->q16;
        skn_ret_args rr = {};
        rr.state = m->state[run]; rr.eps = sp.eps; rr.k_scale = (float)(1.0 / sqrt((double)r.dim)); rr.powers = l.powers;
        if (l.rot_r >= 0) rr.rot = skn_rot{m->rots[l.rot_r].table, r.rot_dims / 2, r.rot_dims / 2};
        rr.q = m->proj + (int64_t)a.heads * a.dim + (int64_t)a.kv_heads * (a.dim + a.vdim);
        rr.k = rr.q + (int64_t)r.heads * r.dim; rr.v = rr.k + (int64_t)r.heads * r.dim; rr.g = rr.v + (int64_t)r.heads * r.vdim; rr.ld = m->ldp;
        rr.out_scale = l.spec.right_scale;
        rr.exact = f32;
        rr.chunks = m->ret_chunks;
        const int64_t rc0 = (int64_t)a.heads * a.vdim;
        if (rows32) {
            aa.out = skn_rows_out{m->mix32, m->ldm, nullptr, 0};
            rr.out = skn_rows_out{m->mix32 + rc0, m->ldm, nullptr, 0};
        } else {
            aa.out = skn_rows_out{nullptr, 0, m->mix16, m->ldm};
            rr.out = skn_rows_out{nullptr, 0, m->mix16 + rc0, m->ldm};
        }
        SKN_CUDA(ctx, st.T == 1 ? skn_launch_mix_decode(ctx, st, &aa, &rr, s) : skn_launch_mix_prefill(ctx, st, &aa, &rr, s));
        // output projection into the residual stream (the side gate takes x as bf16 rows on the tensor-core route)
        const bool side = sp.side_dim > 0, side_once = side && M <= SIDE_ROWS && skn_token_side_fits(l.w.side_gate, l.w.side_proj);
        const bool raw = side && !rows32 && !side_once;
        skn_epi eo = to_rows(SKN_EPI_ADD, m->x, ldw, raw && !l.spec.ff ? m->x16 : nullptr, ldw);
        eo.resid = m->x; eo.ld_resid = ldw;
        SKN_CUDA(ctx, linear(m, few, l.w.w_out, M, m->mix32, m->ldm, m->mix16, m->ldm, nullptr, eo));
        // feed-forward
        if (l.spec.ff) {
            if (!few) SKN_CUDA(ctx, skn_launch_norm_rows(m->x, ldw, M, W, sp.eps, nullptr, 0, nullptr, l.norm2, hout, nullptr, 0, nullptr, s));
            SKN_CUDA(ctx, linear(m, few, l.w.up, M, few ? m->x : m->h32, ldw, m->h16, ldw, few ? l.norm2 : nullptr,
                                 to_rows(SKN_EPI_RELU2, rows32 ? m->u32 : nullptr, m->ldf, rows32 ? nullptr : m->u16, m->ldf)));
            skn_epi ed = to_rows(SKN_EPI_ADD, m->x, ldw, raw ? m->x16 : nullptr, ldw);
            ed.resid = m->x; ed.ld_resid = ldw;
            SKN_CUDA(ctx, linear(m, few, l.w.down, M, m->u32, m->ldf, m->u16, m->ldf, nullptr, ed));
        }
        // token side input
        h_ready = false;
        if (side) {
            const int64_t col = (int64_t)m->runs[run] * sp.side_dim;
            if (side_once) {
                SKN_CUDA(ctx, skn_launch_token_side(l.w.side_gate, l.w.side_proj, m->side_embed, col, ids, m->x, ldw, M, l.side_norm, sp.eps, s));
            } else {
                skn_epi eg = to_rows(SKN_EPI_GELU_TABLE, rows32 ? m->g32 : nullptr, m->lds, rows32 ? nullptr : m->g16, m->lds);
                eg.table = reinterpret_cast<const __nv_bfloat16 *>(m->side_embed->d_blocks);
                eg.ld_table = m->side_embed->pitch / 2; eg.table_rows = m->side_embed->n_rows; eg.table_col = col; eg.ids = ids;
                SKN_CUDA(ctx, linear(m, few, l.w.side_gate, M, m->x, ldw, m->x16, ldw, nullptr, eg));
                SKN_CUDA(ctx, linear(m, few, l.w.side_proj, M, m->g32, m->lds, m->g16, m->lds, nullptr, to_rows(SKN_EPI_STORE, m->y32, ldw, nullptr, 0)));
                // y joins the residual stream in the pass that takes the next run's first norm
                h_ready = !few && run + 1 < m->runs.size() && !m->pass_start[run + 1];
                SKN_CUDA(ctx, skn_launch_norm_rows(m->x, ldw, M, W, sp.eps, m->y32, ldw, l.side_norm, h_ready ? m->layers[m->runs[run + 1]].norm1 : nullptr,
                                                   hout, nullptr, 0, nullptr, s));
            }
        }
        if (m->tracing) {
            const size_t at = m->trace.size();
            m->trace.resize(at + (size_t)M * W);
            SKN_CUDA(ctx, cudaMemcpy2DAsync(m->trace.data() + at, (size_t)W * 4, m->x, (size_t)ldw * 4, (size_t)W * 4, M, cudaMemcpyDeviceToHost, s));
            SKN_CUDA(ctx, cudaStreamSynchronize(s));
        }
    }
    return SKN_OK;
}

// logits of n rows of the residual stream (rows: device list, NULL for the first n) into m->logits
static int32_t run_head(skn_lugasun *m, int n, const int32_t *rows) {
    skn_ctx *ctx = m->ctx;
    const bool few = is_few(m, n), rows32 = few || m->dtype == SKN_LUGASUN_F32;
    const skn_rows_out hout = rows32 ? skn_rows_out{m->h32, m->ldw, nullptr, 0} : skn_rows_out{nullptr, 0, m->h16, m->ldw};
    const bool fold = few && !rows;
    if (!fold)
        SKN_CUDA(ctx, skn_launch_norm_rows(m->x, m->ldw, n, m->spec.width, m->spec.eps, nullptr, 0, nullptr, m->final_norm, hout, nullptr, 0, rows, ctx->stream));
    SKN_CUDA(ctx, linear(m, few, m->embed, n, fold ? m->x : m->h32, m->ldw, m->h16, m->ldw, fold ? m->final_norm : nullptr,
                         to_rows(SKN_EPI_STORE, m->logits, m->spec.vocab, nullptr, 0)));
    return SKN_OK;
}

// the last row of every sequence of the step
__global__ void skn_last_rows_kernel(int32_t *rows, int n, int T) {
    for (int i = threadIdx.x; i < n; i += blockDim.x) rows[i] = i * T + T - 1;
}

extern "C" {

int32_t skn_lugasun_create(skn_ctx *ctx, const skn_lugasun_spec *spec, int32_t max_seqs, int32_t max_tokens, int32_t max_ctx,
                           int32_t dtype, skn_lugasun **out) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!out || !spec) return skn_fail(ctx, SKN_ERR_ARG, "NULL argument");
    *out = nullptr;
    if (dtype != SKN_LUGASUN_F32 && dtype != SKN_LUGASUN_BF16) return skn_fail(ctx, SKN_ERR_TYPE, "unknown decoder number format %d", dtype);
    if (max_seqs < 1 || max_tokens < max_seqs || max_ctx < 1) return skn_fail(ctx, SKN_ERR_ARG, "max_tokens must hold one token of each of max_seqs sequences");
    int32_t rc = check_spec(ctx, spec);
    if (rc) return rc;
    skn_lugasun *m = new (std::nothrow) skn_lugasun();
    if (!m) return skn_fail(ctx, SKN_ERR_OOM, "host allocation failed");
    m->magic = SKN_MAGIC_LUGASUN;
    m->ctx = ctx;
    m->spec = *spec;
    m->max_seqs = max_seqs; m->max_tokens = max_tokens; m->max_ctx = max_ctx; m->dtype = dtype;
    m->matvec_ok = true;
    m->layers.resize(spec->n_layers);
    for (int i = 0; i < spec->n_layers; ++i) {
        Layer &l = m->layers[i];
        l = Layer{};
        l.spec = spec->layers[i];
        l.decay.assign(l.spec.right.decay, l.spec.right.decay + l.spec.right.heads);
        l.spec.right.decay = nullptr;
        l.rot_l = find_rot(m, l.spec.left.rot_base, l.spec.left.rot_dims);
        l.rot_r = find_rot(m, l.spec.right.rot_base, l.spec.right.rot_dims);
    }
    m->spec.layers = nullptr;
    const int a = spec->loop_times ? spec->loop_start : 0, b = spec->loop_times ? spec->loop_stop : 0;
    for (int i = 0; i < a; ++i) { m->runs.push_back(i); m->pass_start.push_back(0); }
    for (int t = 0; t < spec->loop_times; ++t)
        for (int i = a; i < b; ++i) { m->runs.push_back(i); m->pass_start.push_back(i == a); }
    for (int i = b; i < spec->n_layers; ++i) { m->runs.push_back(i); m->pass_start.push_back(0); }
    m->host_pos.assign(max_seqs, 0);
    cudaError_t e = cudaSetDevice(ctx->device);
    for (size_t i = 0; i < m->runs.size() && rc == SKN_OK; ++i) {
        const skn_lugasun_layer &l = m->layers[m->runs[i]].spec;
        // a chunk and one step's tokens, or the whole context
        const int64_t span = (int64_t)l.left.chunk + max_tokens;
        const int cap = l.left.chunk > 0 && span < max_ctx ? (int)span : max_ctx;
        skn_kvcache *kv = nullptr;
        skn_state *state = nullptr;
        rc = skn_kv_create_by_position(ctx, max_seqs, l.left.kv_heads, l.left.dim, l.left.vdim, cap,
                                       dtype == SKN_LUGASUN_F32 ? SKN_KV_F32 : SKN_KV_BF16, &kv);
        if (rc == SKN_OK) m->kv.push_back(kv);
        if (rc == SKN_OK) rc = skn_state_create(ctx, max_seqs, l.right.heads, l.right.dim, l.right.vdim, &state);
        if (rc == SKN_OK) m->state.push_back(state);
    }
    if (rc == SKN_OK) {
        if (e == cudaSuccess) e = allocate(m);
        if (e == cudaSuccess) e = cudaStreamSynchronize(ctx->stream);
        if (e != cudaSuccess) rc = skn_check_cuda(ctx, e, "decoder buffers");
    }
    if (rc != SKN_OK) {
        skn_lugasun_destroy(m);
        return rc;
    }
    *out = m;
    return SKN_OK;
}

int32_t skn_lugasun_destroy(skn_lugasun *m) {
    if (!m || m->magic != SKN_MAGIC_LUGASUN) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    if (skn_ctx_ok(m->ctx)) {
        cudaSetDevice(m->ctx->device);
        cudaStreamSynchronize(m->ctx->stream);
    }
    for (void *p : m->owned) cudaFree(p);
    for (skn_kvcache *k : m->kv) skn_kv_destroy(k);
    for (skn_state *s : m->state) skn_state_destroy(s);
    m->magic = 0;
    delete m;
    return SKN_OK;
}

int32_t skn_lugasun_set_layer(skn_lugasun *m, int32_t layer, const skn_lugasun_weights *w) {
    if (!lug_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    if (layer < 0 || layer >= m->spec.n_layers || !w) return skn_fail(ctx, SKN_ERR_ARG, "layer index out of range");
    Layer &l = m->layers[layer];
    const int W = m->spec.width, F = l.spec.ff, S = m->spec.side_dim;
    if (!w->norm1 || !w->q_gain || !w->k_gain || (F && !w->norm2) || (S && !w->side_norm)) return skn_fail(ctx, SKN_ERR_ARG, "NULL gain");
    if (!dense_is(w->w_in, ctx, in_rows(l.spec), W) || !dense_is(w->w_out, ctx, W, out_cols(l.spec)) ||
        (F && (!dense_is(w->up, ctx, F, W) || !dense_is(w->down, ctx, W, F))) ||
        (S && (!dense_is(w->side_gate, ctx, S, W) || !dense_is(w->side_proj, ctx, W, S))))
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    l.w = *w;
    int32_t rc = put_gain(m, l.norm1, w->norm1, W);
    if (!rc && F) rc = put_gain(m, l.norm2, w->norm2, W);
    if (!rc) rc = put_gain(m, l.q_gain, w->q_gain, l.spec.left.dim);
    if (!rc) rc = put_gain(m, l.k_gain, w->k_gain, l.spec.left.dim);
    if (!rc && S) rc = put_gain(m, l.side_norm, w->side_norm, W);
    m->matvec_ok = m->matvec_ok && fits_matvec(w->w_in) && fits_matvec(w->w_out) && (!F || fits_matvec(w->down));
    return rc;
}

int32_t skn_lugasun_set_head(skn_lugasun *m, const skn_tensor *embed, const float *final_norm_host, const skn_tensor *loop_in,
                             const skn_tensor *side_embed) {
    if (!lug_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    const skn_lugasun_spec &s = m->spec;
    if (!final_norm_host) return skn_fail(ctx, SKN_ERR_ARG, "NULL gain");
    if (!dense_is(embed, ctx, s.vocab, s.width) || (s.loop_times && !dense_is(loop_in, ctx, s.width, 2 * (int64_t)s.width)) ||
        (s.side_dim && !dense_is(side_embed, ctx, s.vocab, (int64_t)s.n_layers * s.side_dim)))
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    m->embed = embed;
    m->loop_in = s.loop_times ? loop_in : nullptr;
    m->side_embed = s.side_dim ? side_embed : nullptr;
    m->matvec_ok = m->matvec_ok && fits_matvec(m->loop_in);
    return put_gain(m, m->final_norm, final_norm_host, s.width);
}

int32_t skn_lugasun_reset(skn_lugasun *m, int32_t seq) {
    if (!lug_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
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

int32_t skn_lugasun_position(const skn_lugasun *m, int32_t seq) {
    return lug_ok(m) && seq >= 0 && seq < m->max_seqs ? m->host_pos[seq] : -1;
}

static int32_t check_forward(skn_lugasun *m, int32_t seq0, int32_t n_seqs, bool tokens, int32_t T) {
    skn_ctx *ctx = m->ctx;
    if (seq0 < 0 || n_seqs < 1 || n_seqs > HEAD_ROWS || seq0 + n_seqs > m->max_seqs) return skn_fail(ctx, SKN_ERR_ARG, "sequences outside the decoder");
    if (T < 1 || (int64_t)n_seqs * T > m->max_tokens) return skn_fail(ctx, SKN_ERR_SHAPE, "a step holds at most %d tokens", m->max_tokens);
    if (!tokens && T != 1) return skn_fail(ctx, SKN_ERR_ARG, "tokens may be NULL only for single-token steps");
    for (int s = seq0; s < seq0 + n_seqs; ++s)
        if (m->host_pos[s] + T > m->max_ctx) return skn_fail(ctx, SKN_ERR_SHAPE, "context of %d tokens exceeded", m->max_ctx);
    if (!m->embed) return skn_fail(ctx, SKN_ERR_ARG, "model head not set");
    for (auto &l : m->layers)
        if (!l.w.w_in) return skn_fail(ctx, SKN_ERR_ARG, "a layer has no weights");
    return SKN_OK;
}

int32_t skn_lugasun_forward_dev(skn_lugasun *m, int32_t seq0, int32_t n_seqs, const int32_t *tokens_dev, int32_t T, int32_t head) {
    if (!lug_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
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
    rc = run_layers(m, st, tokens_dev ? tokens_dev : m->ids_out + seq0);
    if (rc == SKN_OK) {
        const cudaError_t e = skn_launch_advance(st, m->pos, ctx->d_status, ctx->stream);
        if (e != cudaSuccess) rc = skn_check_cuda(ctx, e, "advance");
    }
    if (rc == SKN_OK)
        for (int s = seq0; s < seq0 + n_seqs; ++s) m->host_pos[s] += T;
    if (rc == SKN_OK && head) {
        if (T > 1) skn_last_rows_kernel<<<1, 64, 0, ctx->stream>>>(m->want, n_seqs, T);
        rc = run_head(m, n_seqs, T > 1 ? m->want : nullptr);
        if (rc == SKN_OK) {
            const cudaError_t e = skn_launch_argmax(m->logits, n_seqs, m->spec.vocab, m->ids_out + seq0, m->argmax_scratch, ctx->stream);
            if (e != cudaSuccess) rc = skn_check_cuda(ctx, e, "argmax");
        }
    }
    return rc;
}

int32_t skn_lugasun_forward(skn_lugasun *m, int32_t seq0, int32_t n_seqs, const int32_t *tokens_host, int32_t T, int32_t n_want,
                            const int32_t *want_rows_host, float *logits_host, int32_t *next_host) {
    if (!lug_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    int32_t rc = check_forward(m, seq0, n_seqs, tokens_host != nullptr, T);
    if (rc) return rc;
    if (n_want < 0 || n_want > n_seqs * T || (n_want && (!want_rows_host || !logits_host))) return skn_fail(ctx, SKN_ERR_ARG, "bad list of wanted rows");
    for (int i = 0; i < n_want; ++i)
        if (want_rows_host[i] < 0 || want_rows_host[i] >= n_seqs * T) return skn_fail(ctx, SKN_ERR_ARG, "a wanted row lies outside the step");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    if (tokens_host) SKN_CUDA(ctx, cudaMemcpyAsync(m->ids_in, tokens_host, sizeof(int32_t) * n_seqs * T, cudaMemcpyHostToDevice, ctx->stream));
    rc = skn_lugasun_forward_dev(m, seq0, n_seqs, tokens_host ? m->ids_in : nullptr, T, next_host != nullptr);
    if (rc == SKN_OK && next_host)
        SKN_CUDA(ctx, cudaMemcpyAsync(next_host, m->ids_out + seq0, sizeof(int32_t) * n_seqs, cudaMemcpyDeviceToHost, ctx->stream));
    for (int i = 0; i < n_want && rc == SKN_OK; i += HEAD_ROWS) {
        const int n = n_want - i < HEAD_ROWS ? n_want - i : HEAD_ROWS;
        SKN_CUDA(ctx, cudaMemcpyAsync(m->want, want_rows_host + i, sizeof(int32_t) * n, cudaMemcpyHostToDevice, ctx->stream));
        rc = run_head(m, n, m->want);
        if (rc == SKN_OK)
            SKN_CUDA(ctx, cudaMemcpyAsync(logits_host + (size_t)i * m->spec.vocab, m->logits, sizeof(float) * n * m->spec.vocab, cudaMemcpyDeviceToHost, ctx->stream));
    }
    return rc ? rc : skn_sync(ctx);
}

int32_t skn_lugasun_trace(skn_lugasun *m, int32_t on, int32_t rows, float *out_host) {
    if (!lug_ok(m)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    m->tracing = on != 0;
    if (!out_host) return SKN_OK;
    const size_t n = m->runs.size() * (size_t)rows * m->spec.width;
    if (rows != m->trace_rows || m->trace.size() != n) return skn_fail(ctx, SKN_ERR_ARG, "the last step recorded %d rows", m->trace_rows);
    memcpy(out_host, m->trace.data(), n * sizeof(float));
    return SKN_OK;
}

}  // extern "C"
