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
#include "skn_decoder.cuh"
#include "skn_ptx.cuh"

#include <math.h>
#include <new>
#include <stdlib.h>

namespace {

struct Layer {
    skn_lugasun_layer spec;
    std::vector<double> decay;
    skn_lugasun_weights w;                       // tensors (gains below, on the device)
    float *norm1, *norm2, *q_gain, *k_gain, *side_norm, *powers;
    int rot_l, rot_r;                            // index of the rotation table, -1: none
};

constexpr int SIDE_ROWS = 16;                    // rows whose token side input takes one launch

struct Lugasun : skn_decoder {
    skn_lugasun_spec spec;
    std::vector<Layer> layers;
    const skn_tensor *loop_in, *side_embed;
    // activations; row pitches: joint projection, mixer output, feed-forward, side
    int64_t ldp, ldm, ldf, lds;
    float *xa, *xb, *xalt;                       // the residual stream alternates between two buffers where a pass of the loop starts
    float *x0, *proj, *mix32, *u32, *g32, *y32;
    __nv_bfloat16 *mix16, *u16, *g16, *cat16, *x16, *q16;
    float *attn_scratch, *ret_chunks;
    unsigned *tickets;

    bool ready() const override {
        for (auto &l : layers)
            if (!l.w.w_in) return false;
        return true;
    }
    int32_t run_layers(const skn_step &st, const int32_t *ids) override;
};

}

static Lugasun *lug(skn_decoder *m) { return skn_decoder_ok(m) && m->kind == SKN_KIND_LUGASUN ? static_cast<Lugasun *>(m) : nullptr; }

static int64_t in_rows(const skn_lugasun_layer &l) {
    return (int64_t)l.left.heads * l.left.dim + (int64_t)l.left.kv_heads * (l.left.dim + l.left.vdim) +
           (int64_t)l.right.heads * (2 * l.right.dim + 2 * l.right.vdim);
}
static int64_t out_cols(const skn_lugasun_layer &l) { return (int64_t)l.left.heads * l.left.vdim + (int64_t)l.right.heads * l.right.vdim; }

static int32_t check_spec(skn_ctx *ctx, const skn_lugasun_spec *s) {
    if (s->side_dim < 0 || !s->layers) return skn_fail(ctx, SKN_ERR_ARG, "invalid model geometry");
    for (int i = 0; i < s->n_layers; ++i) {
        int32_t rc = skn_check_attn_spec(ctx, &s->layers[i].left);
        if (!rc) rc = skn_check_retention_spec(ctx, &s->layers[i].right);
        if (rc) return rc;
        if (s->layers[i].ff < 0) return skn_fail(ctx, SKN_ERR_ARG, "negative feed-forward width");
    }
    return SKN_OK;
}

static cudaError_t allocate(Lugasun *m) {
    const skn_lugasun_spec &s = m->spec;
    const bool f32 = m->f32();
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
        const size_t rows = skn_chunk_attn_tc(m->caches[i]) ? (size_t)m->max_seqs : R;
        const size_t a = skn_attn_scratch((int)rows, l.left.heads, l.left.vdim, l.left.chunk, m->max_ctx);
        scratch = a > scratch ? a : scratch;
        tick = rows * l.left.heads > tick ? rows * l.left.heads : tick;
        const size_t c = max_chunks * l.right.heads * l.right.dim * m->states[i]->v_pitch;
        chunks = c > chunks ? c : chunks;
        const size_t q = R * l.left.heads * m->caches[i]->k_pitch;
        if (skn_chunk_attn_tc(m->caches[i]) && q > q16) q16 = q;
    }
    m->ldp = skn_up8(P); m->ldm = skn_up8(X); m->ldf = skn_up8(F); m->lds = skn_up8(s.side_dim);
    const int64_t ldc = skn_up8(2 * (int64_t)s.width);
    cudaError_t e = skn_decoder_allocate(m);
#define LUG_TAKE(p, n) if (e == cudaSuccess) e = m->take(&m->p, n)
    LUG_TAKE(xa, R * m->ldw); LUG_TAKE(xb, R * m->ldw); LUG_TAKE(x0, R * m->ldw);
    LUG_TAKE(proj, R * m->ldp);
    LUG_TAKE(mix32, r32 * m->ldm); LUG_TAKE(u32, r32 * m->ldf); LUG_TAKE(g32, r32 * m->lds);
    LUG_TAKE(y32, s.side_dim ? R * m->ldw : 0);
    LUG_TAKE(mix16, r16 * m->ldm); LUG_TAKE(u16, r16 * m->ldf); LUG_TAKE(g16, r16 * m->lds);
    LUG_TAKE(cat16, s.loop_times ? r16 * ldc : 0); LUG_TAKE(x16, s.side_dim ? r16 * m->ldw : 0); LUG_TAKE(q16, q16);
    LUG_TAKE(attn_scratch, scratch); LUG_TAKE(tickets, tick); LUG_TAKE(ret_chunks, chunks);
#undef LUG_TAKE
    for (auto &l : m->layers) {
        if (e == cudaSuccess) e = m->take(&l.norm1, s.width);
        if (e == cudaSuccess) e = m->take(&l.norm2, s.width);
        if (e == cudaSuccess) e = m->take(&l.side_norm, s.width);
        if (e == cudaSuccess) e = m->take(&l.q_gain, l.spec.left.dim);
        if (e == cudaSuccess) e = m->take(&l.k_gain, l.spec.left.dim);
        const size_t np = (size_t)l.spec.right.heads * (SKN_RET_CHUNK + 1);
        if (e == cudaSuccess) e = m->take(&l.powers, np);
        if (e == cudaSuccess) {
            std::vector<float> pw(np);
            skn_decay_powers(l.decay.data(), l.spec.right.heads, pw.data());
            e = cudaMemcpyAsync(l.powers, pw.data(), np * sizeof(float), cudaMemcpyHostToDevice, m->ctx->stream);
            if (e == cudaSuccess) e = cudaStreamSynchronize(m->ctx->stream);
        }
    }
    return e;
}

// the step's layers; leaves the residual stream in m->x
int32_t Lugasun::run_layers(const skn_step &st, const int32_t *ids) {
    cudaStream_t s = ctx->stream;
    const skn_lugasun_spec &sp = spec;
    const int M = st.n_seqs * st.T, W = sp.width;
    const bool few = this->few(M), rows32 = few || f32();
    x = xa;
    xalt = xb;
    SKN_CUDA(ctx, skn_launch_embed_bf16(embed, ids, M, x, sp.loop_times ? x0 : nullptr, ldw, s));
    SKN_CUDA(ctx, step_angles(st));
    const skn_rows_out hout = h_rows(rows32);
    bool h_ready = false;                        // the first norm of this run was written by the run before
    for (size_t run = 0; run < runs.size(); ++run) {
        Layer &l = layers[runs[run]];
        if (pass[run] >= 0) {
            // x <- W_in [x; x0]
            skn_linear in = {};
            in.w = loop_in;
            in.M = M;
            in.epi = skn_to_rows(SKN_EPI_STORE, xalt, ldw, nullptr, 0);
            if (rows32) {
                in.x32 = x; in.ld_x32 = ldw; in.x32b = x0; in.ld_x32b = ldw; in.k_a = W;
                SKN_CUDA(ctx, launch_linear(few, in));
            } else {
                const int64_t ldc = skn_up8(2 * (int64_t)W);
                SKN_CUDA(ctx, skn_launch_concat_bf16(x, x0, ldw, M, W, cat16, ldc, s));
                in.x16 = cat16; in.ld_x16 = ldc;
                SKN_CUDA(ctx, launch_linear(few, in));
            }
            float *t = x; x = xalt; xalt = t;
            h_ready = false;
        }
        // mixer
        if (!few && !h_ready) SKN_CUDA(ctx, skn_launch_norm_rows(x, ldw, M, W, sp.eps, nullptr, 0, nullptr, l.norm1, hout, nullptr, 0, nullptr, s));
        const skn_attn_spec &a = l.spec.left;
        const skn_retention_spec &r = l.spec.right;
        SKN_CUDA(ctx, linear(few, l.w.w_in, M, few ? x : h32, ldw, h16, ldw, few ? l.norm1 : nullptr,
                             skn_to_rows(SKN_EPI_STORE, proj, ldp, nullptr, 0)));
        skn_attn_args aa = {};
        aa.kv = caches[run]; aa.heads = a.heads; aa.chunk = a.chunk; aa.scale = a.scale; aa.softcap = a.softcap; aa.eps = sp.eps;
        aa.q_gain = l.q_gain; aa.k_gain = l.k_gain;
        aa.rot = rot(l.rot_l);
        aa.q = proj; aa.k = aa.q + (int64_t)a.heads * a.dim; aa.v = aa.k + (int64_t)a.kv_heads * a.dim; aa.ld = ldp;
        aa.out_scale = l.spec.left_scale;
        aa.scratch = attn_scratch; aa.tickets = tickets; aa.q16 = q16;
        skn_ret_args rr = {};
        rr.state = states[run]; rr.eps = sp.eps; rr.k_scale = (float)(1.0 / sqrt((double)r.dim)); rr.powers = l.powers;
        rr.rot = rot(l.rot_r);
        rr.q = proj + (int64_t)a.heads * a.dim + (int64_t)a.kv_heads * (a.dim + a.vdim);
        rr.k = rr.q + (int64_t)r.heads * r.dim; rr.v = rr.k + (int64_t)r.heads * r.dim; rr.g = rr.v + (int64_t)r.heads * r.vdim; rr.ld = ldp;
        rr.out_scale = l.spec.right_scale;
        rr.exact = f32();
        rr.chunks = ret_chunks;
        const int64_t rc0 = (int64_t)a.heads * a.vdim;
        if (rows32) {
            aa.out = skn_rows_out{mix32, ldm, nullptr, 0};
            rr.out = skn_rows_out{mix32 + rc0, ldm, nullptr, 0};
        } else {
            aa.out = skn_rows_out{nullptr, 0, mix16, ldm};
            rr.out = skn_rows_out{nullptr, 0, mix16 + rc0, ldm};
        }
        SKN_CUDA(ctx, st.T == 1 ? skn_launch_mix_decode(ctx, st, &aa, &rr, s) : skn_launch_mix_prefill(ctx, st, &aa, &rr, s));
        // output projection into the residual stream (the side gate takes x as bf16 rows on the tensor-core route)
        const bool side = sp.side_dim > 0, side_once = side && M <= SIDE_ROWS && skn_token_side_fits(l.w.side_gate, l.w.side_proj);
        const bool raw = side && !rows32 && !side_once;
        skn_epi eo = skn_to_rows(SKN_EPI_ADD, x, ldw, raw && !l.spec.ff ? x16 : nullptr, ldw);
        eo.resid = x; eo.ld_resid = ldw;
        SKN_CUDA(ctx, linear(few, l.w.w_out, M, mix32, ldm, mix16, ldm, nullptr, eo));
        // feed-forward
        if (l.spec.ff) {
            if (!few) SKN_CUDA(ctx, skn_launch_norm_rows(x, ldw, M, W, sp.eps, nullptr, 0, nullptr, l.norm2, hout, nullptr, 0, nullptr, s));
            SKN_CUDA(ctx, linear(few, l.w.up, M, few ? x : h32, ldw, h16, ldw, few ? l.norm2 : nullptr,
                                 skn_to_rows(SKN_EPI_RELU2, rows32 ? u32 : nullptr, ldf, rows32 ? nullptr : u16, ldf)));
            skn_epi ed = skn_to_rows(SKN_EPI_ADD, x, ldw, raw ? x16 : nullptr, ldw);
            ed.resid = x; ed.ld_resid = ldw;
            SKN_CUDA(ctx, linear(few, l.w.down, M, u32, ldf, u16, ldf, nullptr, ed));
        }
        // token side input
        h_ready = false;
        if (side) {
            const int64_t col = (int64_t)runs[run] * sp.side_dim;
            if (side_once) {
                SKN_CUDA(ctx, skn_launch_token_side(l.w.side_gate, l.w.side_proj, side_embed, col, ids, x, ldw, M, l.side_norm, sp.eps, s));
            } else {
                skn_epi eg = skn_to_rows(SKN_EPI_GELU_TABLE, rows32 ? g32 : nullptr, lds, rows32 ? nullptr : g16, lds);
                eg.table = reinterpret_cast<const __nv_bfloat16 *>(side_embed->d_blocks);
                eg.ld_table = side_embed->pitch / 2; eg.table_rows = side_embed->n_rows; eg.table_col = col; eg.ids = ids;
                SKN_CUDA(ctx, linear(few, l.w.side_gate, M, x, ldw, x16, ldw, nullptr, eg));
                SKN_CUDA(ctx, linear(few, l.w.side_proj, M, g32, lds, g16, lds, nullptr, skn_to_rows(SKN_EPI_STORE, y32, ldw, nullptr, 0)));
                // y joins the residual stream in the pass that takes the next run's first norm
                h_ready = !few && run + 1 < runs.size() && pass[run + 1] < 0;
                SKN_CUDA(ctx, skn_launch_norm_rows(x, ldw, M, W, sp.eps, y32, ldw, l.side_norm, h_ready ? layers[runs[run + 1]].norm1 : nullptr,
                                                   hout, nullptr, 0, nullptr, s));
            }
        }
        if (tracing) {
            const int32_t rc = record_layer(M);
            if (rc) return rc;
        }
    }
    return SKN_OK;
}

extern "C" {

int32_t skn_lugasun_create(skn_ctx *ctx, const skn_lugasun_spec *spec, int32_t max_seqs, int32_t max_tokens, int32_t max_ctx,
                           int32_t dtype, skn_decoder **out) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!out || !spec) return skn_fail(ctx, SKN_ERR_ARG, "NULL argument");
    *out = nullptr;
    const skn_decoder_sizes sizes = {spec->n_layers, spec->width, spec->vocab, spec->loop_start, spec->loop_stop, spec->loop_times,
                                     max_seqs, max_tokens, max_ctx, dtype, spec->eps};
    int32_t rc = skn_decoder_check(ctx, sizes);
    if (!rc) rc = check_spec(ctx, spec);
    if (rc) return rc;
    Lugasun *m = new (std::nothrow) Lugasun();
    if (!m) return skn_fail(ctx, SKN_ERR_OOM, "host allocation failed");
    skn_decoder_init(m, SKN_KIND_LUGASUN, ctx, sizes);
    m->spec = *spec;
    m->layers.resize(spec->n_layers);
    for (int i = 0; i < spec->n_layers; ++i) {
        Layer &l = m->layers[i];
        l = Layer{};
        l.spec = spec->layers[i];
        l.decay.assign(l.spec.right.decay, l.spec.right.decay + l.spec.right.heads);
        l.spec.right.decay = nullptr;
        l.rot_l = m->find_rot(l.spec.left.rot_base, l.spec.left.rot_dims);
        l.rot_r = m->find_rot(l.spec.right.rot_base, l.spec.right.rot_dims);
    }
    m->spec.layers = nullptr;
    cudaError_t e = cudaSetDevice(ctx->device);
    for (size_t i = 0; i < m->runs.size() && rc == SKN_OK; ++i) {
        const skn_lugasun_layer &l = m->layers[m->runs[i]].spec;
        // a chunk and one step's tokens, or the whole context
        const int64_t span = (int64_t)l.left.chunk + max_tokens;
        const int cap = l.left.chunk > 0 && span < max_ctx ? (int)span : max_ctx;
        skn_kvcache *kv = nullptr;
        skn_state *state = nullptr;
        rc = skn_kv_create_by_position(ctx, max_seqs, l.left.kv_heads, l.left.dim, l.left.vdim, cap,
                                       dtype == SKN_DECODER_F32 ? SKN_KV_F32 : SKN_KV_BF16, &kv);
        if (rc == SKN_OK) m->caches.push_back(kv);
        if (rc == SKN_OK) rc = skn_state_create(ctx, max_seqs, l.right.heads, l.right.dim, l.right.vdim, &state);
        if (rc == SKN_OK) m->states.push_back(state);
    }
    if (rc == SKN_OK) {
        if (e == cudaSuccess) e = allocate(m);
        if (e == cudaSuccess) e = cudaStreamSynchronize(ctx->stream);
        if (e != cudaSuccess) rc = skn_check_cuda(ctx, e, "decoder buffers");
    }
    if (rc != SKN_OK) {
        skn_decoder_destroy(m);
        return rc;
    }
    *out = m;
    return SKN_OK;
}

int32_t skn_lugasun_set_layer(skn_decoder *handle, int32_t layer, const skn_lugasun_weights *w) {
    Lugasun *m = lug(handle);
    if (!m) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    if (layer < 0 || layer >= m->n_layers || !w) return skn_fail(ctx, SKN_ERR_ARG, "layer index out of range");
    Layer &l = m->layers[layer];
    const int W = m->width, F = l.spec.ff, S = m->spec.side_dim;
    if (!w->norm1 || !w->q_gain || !w->k_gain || (F && !w->norm2) || (S && !w->side_norm)) return skn_fail(ctx, SKN_ERR_ARG, "NULL gain");
    if (!skn_dense_is(w->w_in, ctx, in_rows(l.spec), W) || !skn_dense_is(w->w_out, ctx, W, out_cols(l.spec)) ||
        (F && (!skn_dense_is(w->up, ctx, F, W) || !skn_dense_is(w->down, ctx, W, F))) ||
        (S && (!skn_dense_is(w->side_gate, ctx, S, W) || !skn_dense_is(w->side_proj, ctx, W, S))))
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    l.w = *w;
    int32_t rc = skn_put_floats(ctx, l.norm1, w->norm1, W);
    if (!rc && F) rc = skn_put_floats(ctx, l.norm2, w->norm2, W);
    if (!rc) rc = skn_put_floats(ctx, l.q_gain, w->q_gain, l.spec.left.dim);
    if (!rc) rc = skn_put_floats(ctx, l.k_gain, w->k_gain, l.spec.left.dim);
    if (!rc && S) rc = skn_put_floats(ctx, l.side_norm, w->side_norm, W);
    m->matvec_ok = m->matvec_ok && skn_fits_matvec(w->w_in) && skn_fits_matvec(w->w_out) && (!F || skn_fits_matvec(w->down));
    return rc;
}

int32_t skn_lugasun_set_head(skn_decoder *handle, const skn_tensor *embed, const float *final_norm_host, const skn_tensor *loop_in,
                             const skn_tensor *side_embed) {
    Lugasun *m = lug(handle);
    if (!m) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    const skn_lugasun_spec &s = m->spec;
    if (!final_norm_host) return skn_fail(ctx, SKN_ERR_ARG, "NULL gain");
    if (!skn_dense_is(embed, ctx, s.vocab, s.width) || (s.loop_times && !skn_dense_is(loop_in, ctx, s.width, 2 * (int64_t)s.width)) ||
        (s.side_dim && !skn_dense_is(side_embed, ctx, s.vocab, (int64_t)s.n_layers * s.side_dim)))
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    m->embed = embed;
    m->loop_in = s.loop_times ? loop_in : nullptr;
    m->side_embed = s.side_dim ? side_embed : nullptr;
    m->matvec_ok = m->matvec_ok && skn_fits_matvec(m->loop_in);
    return skn_put_floats(ctx, m->final_norm, final_norm_host, s.width);
}

}  // extern "C"
