// The Tutezen decoder over dense bf16 weights: parallel layers, x <- x + m (mixer(h) + feed-forward(h)), h = norm(x), with a selective state space
// or latent attention as the mixer and a dense feed-forward or a mixture of experts beside it.  Everything that reads h is one product, and so
// is everything that adds to x; routes as in skn_decoder.cuh:
//
//   few rows, state space     norm + joint projection (feed-forward's activation in its epilogue) | state update, gate (and routing) |
//                             part norms + joint output + residual
//   few rows, latent          norm + joint projection | norm + query projection | absorbed query, latent into the cache (and routing) |
//                             attention | values and gate | joint output + residual
//   with experts              one launch more (row by row): the chosen experts' gate and up rows; their down rows join the output product
//   more rows                 norm | joint projection | mixer | joint output, and for experts: choice, grouping, two grouped products, sum
#include "skn_decoder.cuh"
#include "skn_latent.cuh"
#include "skn_ssm.cuh"

#include <algorithm>
#include <math.h>
#include <new>

namespace {

constexpr int EXPAND_TOKENS = 32;        // tokens of a sequence from which keys and values are expanded
constexpr int CHUNK_TOKENS = 32;         // tokens of a sequence from which the state space runs in chunks

struct Layer {
    skn_tutezen_layer spec;
    skn_tutezen_weights w;               // tensors (vectors below, on the device)
    float *norm, *conv, *conv_b, *dt_bias, *a, *d, *out_norm, *q_gain, *kv_gain, *sink;
    int rot;
    // padded widths, and the parts of a joint row
    int vp, np, dim, rp, kvp, qr;        // head, state; unrotated, rotated, latent, query latent
    int experts, act;                    // router rows; columns of the dense or shared activation
    int ep;                              // columns of an expert's activation
    int mix_rows, router_at, act_at, in_rows, mix_cols;
};

struct Tutezen : skn_decoder {
    std::vector<Layer> layers;
    std::vector<int> cache_of, state_of;     // per run: its cache, or its state (the convolution's ring is the next one); -1
    float mult;
    int passes;
    float *step;                             // [passes][width]
    int64_t ldp, ldm;                        // pitches: joint projection, output product's input
    float *x0, *proj, *mix32, *y;
    __nv_bfloat16 *mix16;
    // state space
    __nv_bfloat16 *xbc;
    float *dt, *cum, *chunks;
    __nv_bfloat16 *starts;
    // latent attention
    int64_t ldc;
    float *q, *ql, *ol, *scratch, *cq32;
    __nv_bfloat16 *cq16, *q16, *kvx;
    unsigned *tickets;
    // experts
    int64_t lde;
    int32_t *expert, *offset, *place;
    float *weight, *ex32, *ea32, *ey32;      // grouped rows: input, activation, output
    __nv_bfloat16 *ex16, *ea16, *ey16;

    bool ready() const override {
        for (auto &l : layers)
            if (!l.w.w_in) return false;
        return true;
    }
    int32_t run_layers(const skn_step &st, const int32_t *ids) override;
    int32_t ssm_mixer(const Layer &l, const skn_step &st, int run, bool few_rows, const skn_route_args &route);
    int32_t latent_mixer(const Layer &l, const skn_step &st, int run, bool few_rows, const skn_route_args &route);
    int32_t output_few(const Layer &l, int M);
    int32_t output_many(const Layer &l, int M);
};

inline int up8(int n) { return (n + 7) / 8 * 8; }
template <class T> void grow(T &a, T b) { a = b > a ? b : a; }

void lay_out(Layer &l) {
    const skn_tutezen_layer &s = l.spec;
    if (s.mixer == SKN_MIXER_SSM) {
        l.vp = up8(s.ssm.vdim);
        l.np = up8(s.ssm.state);
        l.mix_cols = s.ssm.heads * l.vp;
        l.mix_rows = l.mix_cols + skn_ssm_channels(s.ssm.heads, l.vp, s.ssm.groups, l.np) + up8(s.ssm.heads);
    } else {
        const skn_latent_spec &a = s.latent;
        l.vp = up8(a.vdim);
        l.dim = up8(a.dim);
        l.rp = (l.dim + a.rot_dim + 15) / 16 * 16 - l.dim;
        l.kvp = up8(a.kv_rank);
        l.qr = up8(a.q_rank);
        l.mix_cols = a.heads * l.vp;
        l.mix_rows = l.qr + l.kvp + l.rp + l.mix_cols;
    }
    l.experts = up8(s.experts);
    l.ep = up8(s.expert_ff);
    l.act = up8(s.experts ? s.shared_ff : s.ff);
    l.router_at = l.mix_rows;
    l.act_at = l.router_at + l.experts;
    l.in_rows = l.act_at + (s.experts ? 2 : 1) * l.act;
}

int32_t check_layer(skn_ctx *ctx, const skn_tutezen_layer &s) {
    int32_t rc = SKN_OK;
    if (s.mixer == SKN_MIXER_SSM) rc = skn_check_ssm_spec(ctx, &s.ssm);
    else if (s.mixer == SKN_MIXER_LATENT) rc = skn_check_latent_spec(ctx, &s.latent);
    else return skn_fail(ctx, SKN_ERR_TYPE, "unknown mixer %d", s.mixer);
    if (rc) return rc;
    if (s.ff < 0 || s.experts < 0 || s.shared_ff < 0 || s.experts > SKN_MAX_EXPERTS ||
        (s.experts && (s.ff || s.top < 1 || s.top > s.experts || s.expert_ff < 1)))
        return skn_fail(ctx, SKN_ERR_ARG, "invalid feed-forward geometry");
    return SKN_OK;
}

}

static Tutezen *tut(skn_decoder *m) { return skn_decoder_ok(m) && m->kind == SKN_KIND_TUTEZEN ? static_cast<Tutezen *>(m) : nullptr; }

static cudaError_t allocate(Tutezen *m) {
    const bool f32 = m->f32();
    const size_t R = m->max_tokens, few = R < SKN_MATVEC_ROWS ? R : SKN_MATVEC_ROWS, r32 = f32 ? R : few, r16 = f32 ? 0 : R;
    const size_t short_rows = std::min(R, (size_t)m->max_seqs * (EXPAND_TOKENS - 1)), max_chunks = R / SKN_SSM_CHUNK + m->max_seqs + 1;
    int64_t P = 0, X = 0, Y = 0, C = 0, E = 0, D = 0;
    size_t xbc = 0, heads = 0, chunks = 0, q = 0, ql = 0, ol = 0, scratch = 1, tick = 1, q16 = 0, kvx = 0, pairs = 0, experts = 0;
    for (size_t i = 0; i < m->runs.size(); ++i) {
        const Layer &l = m->layers[m->runs[i]];
        const skn_tutezen_layer &s = l.spec;
        grow(P, (int64_t)l.in_rows);
        grow(X, (int64_t)l.mix_cols + l.act);
        if (s.mixer == SKN_MIXER_SSM) {
            grow(Y, (int64_t)l.mix_cols);
            if (!f32 && skn_ssm_chunks_fit(l.vp, l.np)) {
                grow(xbc, R * skn_ssm_channels(s.ssm.heads, l.vp, s.ssm.groups, l.np));
                grow(heads, R * s.ssm.heads);
                grow(chunks, max_chunks * s.ssm.heads * l.np * l.vp);
            }
        } else {
            const skn_latent_spec &a = s.latent;
            const skn_kvcache *kv = m->caches[m->cache_of[i]];
            grow(C, (int64_t)l.qr);
            skn_latent_args la = {};
            la.kv = kv; la.heads = a.heads; la.dim = l.dim; la.rp = l.rp; la.vdim = l.vp; la.kvp = l.kvp; la.window = a.window;
            const bool expand = skn_latent_expand_fits(la);
            const size_t rows = expand ? short_rows : R;             // rows that meet the absorbed form
            grow(q, rows * a.heads * (l.dim + l.rp));
            grow(ql, rows * a.heads * (l.kvp + l.rp));
            grow(ol, rows * a.heads * l.kvp);
            grow(scratch, skn_latent_scratch(la, (int)rows, m->max_ctx));
            grow(tick, rows * a.heads);
            if (expand) {
                grow(q16, R * a.heads * (l.dim + l.rp));
                grow(kvx, (size_t)kv->capacity * a.heads * (l.dim + l.vp));
            }
        }
        if (s.experts) {
            grow(E, (int64_t)l.ep);
            grow(pairs, R * s.top);
            grow(experts, (size_t)s.experts);
            grow(D, (int64_t)s.top * l.ep);
        }
    }
    m->ldp = P; m->ldm = X; m->ldc = C; m->lde = E;
    cudaError_t e = skn_decoder_allocate(m);
#define TUT_TAKE(p, n) if (e == cudaSuccess) e = m->take(&m->p, n)
    TUT_TAKE(x, R * m->ldw); TUT_TAKE(x0, m->passes > 1 ? R * m->ldw : 0); TUT_TAKE(step, (size_t)m->passes * m->width);
    TUT_TAKE(proj, R * P); TUT_TAKE(mix32, r32 * X); TUT_TAKE(mix16, r16 * X); TUT_TAKE(y, R * Y);
    TUT_TAKE(xbc, xbc); TUT_TAKE(dt, heads); TUT_TAKE(cum, heads); TUT_TAKE(chunks, chunks); TUT_TAKE(starts, 2 * chunks);
    TUT_TAKE(q, q); TUT_TAKE(ql, ql); TUT_TAKE(ol, ol); TUT_TAKE(scratch, scratch); TUT_TAKE(tickets, tick);
    TUT_TAKE(cq32, C ? r32 * C : 0); TUT_TAKE(cq16, C ? r16 * C : 0); TUT_TAKE(q16, q16); TUT_TAKE(kvx, kvx);
    TUT_TAKE(expert, pairs); TUT_TAKE(weight, pairs); TUT_TAKE(place, pairs); TUT_TAKE(offset, experts ? experts + 1 : 0);
    TUT_TAKE(ex32, f32 ? pairs * m->ldw : 0); TUT_TAKE(ex16, f32 ? 0 : pairs * m->ldw);
    TUT_TAKE(ea32, std::max((size_t)D, f32 ? pairs * E : 0)); TUT_TAKE(ea16, f32 ? 0 : pairs * E);
    TUT_TAKE(ey32, f32 ? pairs * m->ldw : 0); TUT_TAKE(ey16, f32 ? 0 : pairs * m->ldw);
#undef TUT_TAKE
    for (auto &l : m->layers) {
        const skn_tutezen_layer &s = l.spec;
#define TUT_TAKE(p, n) if (e == cudaSuccess) e = m->take(&l.p, n)
        TUT_TAKE(norm, m->width);
        if (s.mixer == SKN_MIXER_SSM) {
            const size_t ch = skn_ssm_channels(s.ssm.heads, l.vp, s.ssm.groups, l.np);
            TUT_TAKE(conv, ch * s.ssm.taps); TUT_TAKE(conv_b, ch);
            TUT_TAKE(dt_bias, s.ssm.heads); TUT_TAKE(a, s.ssm.heads); TUT_TAKE(d, s.ssm.heads); TUT_TAKE(out_norm, l.mix_cols);
        } else {
            TUT_TAKE(q_gain, s.latent.q_rank); TUT_TAKE(kv_gain, s.latent.kv_rank); TUT_TAKE(sink, s.latent.heads);
        }
#undef TUT_TAKE
    }
    return e;
}

int32_t Tutezen::ssm_mixer(const Layer &l, const skn_step &st, int run, bool few_rows, const skn_route_args &route) {
    const skn_ssm_spec &s = l.spec.ssm;
    const int M = st.n_seqs * st.T;
    skn_ssm_args a = {};
    a.state = states[state_of[run]]; a.ring = states[state_of[run] + 1];
    a.heads = s.heads; a.vp = l.vp; a.np = l.np; a.groups = s.groups; a.taps = s.taps;
    a.conv = l.conv; a.conv_b = l.conv_b; a.dt_bias = l.dt_bias; a.a = l.a; a.d = l.d;
    a.proj = proj; a.ld = ldp;
    a.xbc = xbc; a.dt = dt; a.cum = cum; a.chunks = chunks; a.starts = starts;
    if (few_rows) {
        a.y = mix32; a.ld_y = ldm;
        a.route = route;
        SKN_CUDA(ctx, skn_launch_ssm_step(st, a, ctx->stream));
        // (the norms of whole vectors of columns are folded into the output product)
        if (l.vp != s.vdim || !skn_norm_folds(l.mix_cols, s.norm_groups))
            SKN_CUDA(ctx, skn_launch_part_norm_rows(mix32, ldm, M, s.heads, s.vdim, l.vp, s.norm_groups, eps, l.out_norm,
                                                    skn_rows_out{mix32, ldm, nullptr, 0}, ctx->stream));
        return SKN_OK;
    }
    a.y = y; a.ld_y = l.mix_cols;
    if (!f32() && st.T >= CHUNK_TOKENS && skn_ssm_chunks_fit(l.vp, l.np)) SKN_CUDA(ctx, skn_launch_ssm_chunks(st, a, ctx->stream));
    else SKN_CUDA(ctx, skn_launch_ssm_step(st, a, ctx->stream));
    const skn_rows_out out = f32() ? skn_rows_out{mix32, ldm, nullptr, 0} : skn_rows_out{nullptr, 0, mix16, ldm};
    SKN_CUDA(ctx, skn_launch_part_norm_rows(y, l.mix_cols, M, s.heads, s.vdim, l.vp, s.norm_groups, eps, l.out_norm, out, ctx->stream));
    return SKN_OK;
}

int32_t Tutezen::latent_mixer(const Layer &l, const skn_step &st, int run, bool few_rows, const skn_route_args &route) {
    const skn_latent_spec &s = l.spec.latent;
    const int M = st.n_seqs * st.T, qd = s.heads * (l.dim + l.rp);
    skn_latent_args a = {};
    a.kv = caches[cache_of[run]];
    a.heads = s.heads; a.dim = l.dim; a.rp = l.rp; a.vdim = l.vp; a.q_rank = s.q_rank; a.kv_rank = s.kv_rank; a.kvp = l.kvp; a.window = s.window;
    a.scale = s.scale; a.eps = eps;
    a.q_gain = l.q_gain; a.kv_gain = l.kv_gain; a.sink = l.sink;
    a.rot = rot(l.rot);
    a.dq = proj; a.dkv = proj + l.qr; a.gate = a.dkv + l.kvp + l.rp; a.ld = ldp;
    a.uq = l.w.uq; a.ukv = l.w.ukv;
    a.q = q; a.ql = ql; a.ol = ol; a.scratch = scratch; a.tickets = tickets;
    a.q16 = q16; a.kvx = kvx;
    a.out = few_rows || f32() ? skn_rows_out{mix32, ldm, nullptr, 0} : skn_rows_out{nullptr, 0, mix16, ldm};
    if (few_rows) {
        a.route = route;
        SKN_CUDA(ctx, linear(true, a.uq, M, a.dq, ldp, nullptr, 0, l.q_gain, skn_to_rows(SKN_EPI_STORE, q, qd, nullptr, 0)));
        SKN_CUDA(ctx, skn_launch_latent_absorbed(st, a, true, ctx->stream));
        return SKN_OK;
    }
    const bool expand = st.T >= EXPAND_TOKENS && skn_latent_expand_fits(a);
    const skn_rows_out cq = f32() ? skn_rows_out{cq32, ldc, nullptr, 0} : skn_rows_out{nullptr, 0, cq16, ldc};
    SKN_CUDA(ctx, skn_launch_latent_rows(st, a, cq, ctx->stream));
    skn_epi e = expand ? skn_to_rows(SKN_EPI_ROTATE, nullptr, 0, q16, qd) : skn_to_rows(SKN_EPI_STORE, q, qd, nullptr, 0);
    e.rot = a.rot; e.rot_head = l.dim + l.rp; e.rot_lo = l.dim;
    SKN_CUDA(ctx, linear(false, a.uq, M, cq32, ldc, cq16, ldc, nullptr, e));
    if (!expand) {
        SKN_CUDA(ctx, skn_launch_latent_absorbed(st, a, false, ctx->stream));
        return SKN_OK;
    }
    int32_t len[SKN_HEAD_ROWS];
    for (int i = 0; i < st.n_seqs; ++i) len[i] = host_pos[st.slot0 + i] + st.T;
    SKN_CUDA(ctx, skn_launch_latent_expanded(ctx, st, a, len, ws, ctx->stream));
    return SKN_OK;
}

// x += mult * (joint output), experts included: row by row when there are any
int32_t Tutezen::output_few(const Layer &l, int M) {
    const skn_tutezen_layer &s = l.spec;
    skn_linear o = {};
    o.w = l.w.w_out;
    o.M = s.experts ? 1 : M;
    o.ld_x32 = ldm;
    o.eps = eps;
    if (s.mixer == SKN_MIXER_SSM && l.vp == s.ssm.vdim && skn_norm_folds(l.mix_cols, s.ssm.norm_groups)) {
        o.gain = l.out_norm;
        o.norm_cols = l.mix_cols;
        o.norm_parts = s.ssm.norm_groups;
    }
    for (int m = 0; m < M; m += o.M) {
        o.x32 = mix32 + m * ldm;
        o.epi = skn_to_rows(SKN_EPI_ADD, x + m * ldw, ldw, nullptr, 0);
        o.epi.alpha = mult; o.epi.resid = x + m * ldw; o.epi.ld_resid = ldw;
        if (s.experts) {
            skn_linear in = {};
            in.w = l.w.e_in;
            in.M = 1;
            in.x32 = x + m * ldw; in.ld_x32 = ldw;
            in.gain = l.norm; in.eps = eps;
            in.pick = skn_pick{SKN_PICK_ROWS, s.top, expert + m * s.top, nullptr, 2 * l.ep, nullptr};
            in.epi = skn_to_rows(SKN_EPI_SILU_TAIL, nullptr, 0, nullptr, 0);
            in.epi.act32 = ea32;
            in.epi.act_scale = weight + m * s.top; in.epi.scale_rows = 2 * l.ep;
            SKN_CUDA(ctx, launch_linear(true, in));
            o.x32b = ea32; o.ld_x32b = 0; o.k_a = l.w.w_out->n_cols;
            o.pick = skn_pick{SKN_PICK_COLS, s.top, expert + m * s.top, l.w.e_out, 0, nullptr};
        }
        SKN_CUDA(ctx, launch_linear(true, o));
    }
    return SKN_OK;
}

int32_t Tutezen::output_many(const Layer &l, int M) {
    const skn_tutezen_layer &s = l.spec;
    cudaStream_t st = ctx->stream;
    skn_epi e = skn_to_rows(SKN_EPI_ADD, x, ldw, nullptr, 0);
    e.alpha = mult; e.resid = x; e.ld_resid = ldw;
    SKN_CUDA(ctx, linear(false, l.w.w_out, M, mix32, ldm, mix16, ldm, nullptr, e));
    if (!s.experts) return SKN_OK;
    const int pairs = M * s.top;
    SKN_CUDA(ctx, skn_launch_group_pairs(expert, pairs, s.experts, offset, place, st));
    SKN_CUDA(ctx, skn_launch_scatter_rows(h_rows(f32()), M, width, s.top, place, f32() ? skn_rows_out{ex32, ldw, nullptr, 0} : skn_rows_out{nullptr, 0, ex16, ldw}, st));
    skn_linear g = {};
    g.w = l.w.e_in;
    g.M = pairs;
    g.x32 = ex32; g.ld_x32 = ldw; g.x16 = ex16; g.ld_x16 = ldw;
    g.pick = skn_pick{SKN_PICK_GROUPS, s.experts, nullptr, nullptr, 2 * l.ep, offset};
    g.epi = skn_to_rows(SKN_EPI_SILU_TAIL, nullptr, 0, nullptr, 0);
    g.epi.act32 = f32() ? ea32 : nullptr; g.epi.ld_act32 = lde;
    g.epi.act16 = f32() ? nullptr : ea16; g.epi.ld_act16 = lde;
    SKN_CUDA(ctx, launch_linear(false, g));
    g.w = l.w.e_out;
    g.x32 = ea32; g.ld_x32 = lde; g.x16 = ea16; g.ld_x16 = lde;
    g.pick.rows_per = width;
    g.epi = f32() ? skn_to_rows(SKN_EPI_STORE, ey32, ldw, nullptr, 0) : skn_to_rows(SKN_EPI_STORE, nullptr, 0, ey16, ldw);
    SKN_CUDA(ctx, launch_linear(false, g));
    SKN_CUDA(ctx, skn_launch_gather_experts(x, ldw, M, width, mult, s.top, place, weight,
                                            f32() ? skn_rows_out{ey32, ldw, nullptr, 0} : skn_rows_out{nullptr, 0, ey16, ldw}, st));
    return SKN_OK;
}

// the step's layers; leaves the residual stream in x
int32_t Tutezen::run_layers(const skn_step &st, const int32_t *ids) {
    cudaStream_t s = ctx->stream;
    const int M = st.n_seqs * st.T, W = width;
    const bool few_rows = few(M), rows32 = few_rows || f32();
    SKN_CUDA(ctx, skn_launch_embed_bf16(embed, ids, M, x, x0, ldw, s));
    SKN_CUDA(ctx, step_angles(st));
    for (size_t run = 0; run < runs.size(); ++run) {
        const Layer &l = layers[runs[run]];
        const skn_tutezen_layer &sp = l.spec;
        if (pass[run] >= 0)
            SKN_CUDA(ctx, skn_launch_add_vec_rows(x, ldw, M, W, step + (size_t)pass[run] * W, pass[run] > 0 ? x0 : nullptr, ldw, s));
        if (!few_rows)
            SKN_CUDA(ctx, skn_launch_norm_rows(x, ldw, M, W, eps, nullptr, 0, nullptr, l.norm, h_rows(rows32), nullptr, 0, nullptr, s));
        skn_epi e = skn_to_rows(!l.act ? SKN_EPI_STORE : sp.experts ? SKN_EPI_SILU_TAIL : SKN_EPI_GELU_TAIL, proj, ldp, nullptr, 0);
        e.n_act = l.act_at;
        if (rows32) { e.act32 = mix32 + l.mix_cols; e.ld_act32 = ldm; }
        else { e.act16 = mix16 + l.mix_cols; e.ld_act16 = ldm; }
        SKN_CUDA(ctx, linear(few_rows, l.w.w_in, M, few_rows ? x : h32, ldw, h16, ldw, few_rows ? l.norm : nullptr, e));
        skn_route_args route = {};
        if (sp.experts) route = skn_route_args{proj + l.router_at, ldp, sp.experts, sp.top, expert, weight};
        if (sp.experts && !few_rows) SKN_CUDA(ctx, skn_launch_route(route, M, s));
        int32_t rc = sp.mixer == SKN_MIXER_SSM ? ssm_mixer(l, st, (int)run, few_rows, route) : latent_mixer(l, st, (int)run, few_rows, route);
        if (!rc) rc = few_rows ? output_few(l, M) : output_many(l, M);
        if (!rc && tracing) rc = record_layer(M);
        if (rc) return rc;
    }
    return SKN_OK;
}

extern "C" {

int32_t skn_tutezen_create(skn_ctx *ctx, const skn_tutezen_spec *spec, int32_t max_seqs, int32_t max_tokens, int32_t max_ctx, int32_t dtype,
                           skn_decoder **out) {
    if (!skn_ctx_ok(ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad context handle");
    SKN_ENTER(ctx);
    if (!out || !spec || !spec->layers) return skn_fail(ctx, SKN_ERR_ARG, "NULL argument");
    *out = nullptr;
    const skn_decoder_sizes sizes = {spec->n_layers, spec->width, spec->vocab, spec->loop_start, spec->loop_stop, spec->loop_times,
                                     max_seqs, max_tokens, max_ctx, dtype, spec->eps};
    int32_t rc = skn_decoder_check(ctx, sizes);
    for (int i = 0; i < spec->n_layers && !rc; ++i) rc = check_layer(ctx, spec->layers[i]);
    if (rc) return rc;
    Tutezen *m = new (std::nothrow) Tutezen();
    if (!m) return skn_fail(ctx, SKN_ERR_OOM, "host allocation failed");
    skn_decoder_init(m, SKN_KIND_TUTEZEN, ctx, sizes);
    m->mult = spec->residual_mult;
    m->passes = spec->loop_times;
    m->layers.resize(spec->n_layers);
    for (int i = 0; i < spec->n_layers; ++i) {
        Layer &l = m->layers[i];
        l = Layer{};
        l.spec = spec->layers[i];
        l.rot = l.spec.mixer == SKN_MIXER_LATENT ? m->find_rot(l.spec.latent.rot_base, l.spec.latent.rot_dims) : -1;
        lay_out(l);
    }
    cudaError_t e = cudaSetDevice(ctx->device);
    for (size_t i = 0; i < m->runs.size() && rc == SKN_OK; ++i) {
        const Layer &l = m->layers[m->runs[i]];
        m->cache_of.push_back(-1);
        m->state_of.push_back(-1);
        if (l.spec.mixer == SKN_MIXER_SSM) {
            const skn_ssm_spec &s = l.spec.ssm;
            skn_state *state = nullptr, *ring = nullptr;
            m->state_of[i] = (int)m->states.size();
            rc = skn_state_create(ctx, max_seqs, s.heads, l.np, l.vp, &state);
            if (rc == SKN_OK) m->states.push_back(state);
            if (rc == SKN_OK) rc = skn_state_create(ctx, max_seqs, 1, s.taps, skn_ssm_channels(s.heads, l.vp, s.groups, l.np), &ring);
            if (rc == SKN_OK) m->states.push_back(ring);
        } else {
            // a window and one step's tokens, or the whole context
            const int64_t span = (int64_t)l.spec.latent.window + max_tokens;
            const int cap = l.spec.latent.window > 0 && span < max_ctx ? (int)span : max_ctx;
            skn_kvcache *kv = nullptr;
            m->cache_of[i] = (int)m->caches.size();
            rc = skn_kv_create_by_position(ctx, max_seqs, 1, l.kvp + l.rp, 0, cap, dtype == SKN_DECODER_F32 ? SKN_KV_F32 : SKN_KV_BF16, &kv);
            if (rc == SKN_OK) m->caches.push_back(kv);
        }
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

int32_t skn_tutezen_set_layer(skn_decoder *handle, int32_t layer, const skn_tutezen_weights *w) {
    Tutezen *m = tut(handle);
    if (!m) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    if (layer < 0 || layer >= m->n_layers || !w) return skn_fail(ctx, SKN_ERR_ARG, "layer index out of range");
    Layer &l = m->layers[layer];
    const skn_tutezen_layer &s = l.spec;
    const int W = m->width;
    const bool ssm = s.mixer == SKN_MIXER_SSM;
    if (!w->norm || (ssm ? !w->conv || !w->conv_b || !w->dt_bias || !w->a_log || !w->d || !w->out_norm : !w->q_gain || !w->kv_gain || !w->sink))
        return skn_fail(ctx, SKN_ERR_ARG, "NULL vector");
    const int64_t lh = (int64_t)s.latent.heads;
    if (!skn_dense_is(w->w_in, ctx, l.in_rows, W) || !skn_dense_is(w->w_out, ctx, W, l.mix_cols + l.act) ||
        (!ssm && (!skn_dense_is(w->uq, ctx, lh * (l.dim + l.rp), s.latent.q_rank) || !skn_dense_is(w->ukv, ctx, lh * (l.dim + l.vp), s.latent.kv_rank))) ||
        (s.experts && (!skn_dense_is(w->e_in, ctx, (int64_t)s.experts * 2 * l.ep, W) || !skn_dense_is(w->e_out, ctx, (int64_t)s.experts * W, l.ep))))
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    l.w = *w;
    int32_t rc = skn_put_floats(ctx, l.norm, w->norm, W);
    if (ssm) {
        const int H = s.ssm.heads, ch = skn_ssm_channels(H, l.vp, s.ssm.groups, l.np), taps = s.ssm.taps;
        std::vector<float> conv((size_t)ch * taps), a(H);
        for (int c = 0; c < ch; ++c)
            for (int k = 0; k < taps; ++k) conv[(size_t)k * ch + c] = w->conv[(size_t)c * taps + k];
        for (int h = 0; h < H; ++h) a[h] = -expf(w->a_log[h]);
        if (!rc) rc = skn_put_floats(ctx, l.conv, conv.data(), conv.size());
        if (!rc) rc = skn_put_floats(ctx, l.conv_b, w->conv_b, ch);
        if (!rc) rc = skn_put_floats(ctx, l.dt_bias, w->dt_bias, H);
        if (!rc) rc = skn_put_floats(ctx, l.a, a.data(), H);
        if (!rc) rc = skn_put_floats(ctx, l.d, w->d, H);
        if (!rc) rc = skn_put_floats(ctx, l.out_norm, w->out_norm, l.mix_cols);
    } else {
        if (!rc) rc = skn_put_floats(ctx, l.q_gain, w->q_gain, s.latent.q_rank);
        if (!rc) rc = skn_put_floats(ctx, l.kv_gain, w->kv_gain, s.latent.kv_rank);
        if (!rc) rc = skn_put_floats(ctx, l.sink, w->sink, s.latent.heads);
    }
    bool fits = skn_fits_matvec(w->w_in) && skn_fits_matvec(w->w_out) && (ssm || skn_fits_matvec(w->uq));
    if (s.experts) fits = fits && skn_fits_matvec(w->e_in) && w->w_out->pitch + s.top * w->e_out->pitch <= 64 * 1024;
    m->matvec_ok = m->matvec_ok && fits;
    return rc;
}

int32_t skn_tutezen_set_head(skn_decoder *handle, const skn_tensor *embed, const float *final_norm_host, const float *loop_step_host) {
    Tutezen *m = tut(handle);
    if (!m) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad decoder handle");
    skn_ctx *ctx = m->ctx;
    SKN_ENTER(ctx);
    if (!final_norm_host || (m->passes && !loop_step_host)) return skn_fail(ctx, SKN_ERR_ARG, "NULL vector");
    if (!skn_dense_is(embed, ctx, m->vocab, m->width)) return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    m->embed = embed;
    int32_t rc = skn_put_floats(ctx, m->final_norm, final_norm_host, m->width);
    if (!rc && m->passes) rc = skn_put_floats(ctx, m->step, loop_step_host, (size_t)m->passes * m->width);
    return rc;
}

}  // extern "C"
