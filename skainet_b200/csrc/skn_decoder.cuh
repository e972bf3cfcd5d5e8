// What the decoders over dense bf16 weights share: sequences in slots with positions of their own, the order in which
// layers run (a range of them may be looped), step buffers, rotation tables, the three routes of a linear layer, the
// output layer, and the recording of the residual stream.  A model derives from skn_decoder and supplies its layers.
//
//   few rows                fp32 activations on the matvec kernel, RMS norms folded in
//   bf16, more rows         tcgen05 products of bf16 rows, norms as row kernels
//   fp32, more rows         the same sequence with fp32 rows and fp32 products
//
// The residual stream is fp32 in every route.  A step is a fixed sequence of launches on the context's stream, all with
// programmatic dependent launch and capturable in a CUDA graph.
#pragma once
#include "skn_mixers.cuh"

#include <vector>

#define SKN_MAGIC_DECODER 0x736b6e75u   // 'sknu'
constexpr int SKN_HEAD_ROWS = 64;       // rows of logits computed at a time; sequences of one step

static inline int64_t skn_up8(int64_t n) { return (n + 7) / 8 * 8; }

struct skn_rot_entry {
    double base;
    int dims;
    double *freq;
    float2 *table;                      // angles of the step, [max_tokens][dims / 2]
};

struct skn_decoder {
    uint32_t magic;
    int kind;                           // which model (skn_decoder_kind)
    skn_ctx *ctx;
    int32_t max_seqs, max_tokens, max_ctx, dtype, n_layers;
    int width, vocab;
    float eps;
    std::vector<int> runs;              // layer index of every layer run
    std::vector<int> pass;              // number of the loop's pass that begins before a run, -1: none
    std::vector<skn_kvcache *> caches;  // owned
    std::vector<skn_state *> states;    // owned
    std::vector<skn_rot_entry> rots;
    std::vector<void *> owned;          // device allocations
    const skn_tensor *embed;
    float *final_norm;
    std::vector<int32_t> host_pos;
    int32_t *pos, *ids_in, *ids_out, *want;
    bool matvec_ok;                     // every weight's row fits the matvec kernel
    int64_t ldw;                        // pitch of rows of the model width
    float *x;                           // residual stream of the last step
    float *h32, *logits;
    __nv_bfloat16 *h16;
    skn_dense_ws ws;
    void *argmax_scratch;
    bool tracing;
    std::vector<float> trace;
    int trace_rows;

    virtual ~skn_decoder() {}
    virtual bool ready() const = 0;     // every layer has its weights
    // the step's layers; leaves the residual stream in x
    virtual int32_t run_layers(const skn_step &st, const int32_t *ids) = 0;

    bool f32() const;
    bool few(int rows) const;           // rows of a step that take the matvec route
    // where normalised rows go in the many-row routes
    skn_rows_out h_rows(bool rows32) const { return rows32 ? skn_rows_out{h32, ldw, nullptr, 0} : skn_rows_out{nullptr, 0, h16, ldw}; }
    template <class T> cudaError_t take(T **p, size_t n) {
        *p = nullptr;
        if (n == 0) return cudaSuccess;
        const cudaError_t e = cudaMalloc((void **)p, n * sizeof(T));
        if (e != cudaSuccess) return e;
        owned.push_back(*p);
        return cudaMemsetAsync(*p, 0, n * sizeof(T), ctx->stream);      // row padding stays zero
    }
    int find_rot(double base, int dims);                // index of the rotation table, -1 for dims == 0
    skn_rot rot(int i) const { return i < 0 ? skn_rot{nullptr, 0, 0} : skn_rot{rots[i].table, rots[i].dims / 2, rots[i].dims / 2}; }
    cudaError_t step_angles(const skn_step &st);        // fills the rotation tables
    // The routes of a linear layer.  in32 / in16: the same rows in either form (in16 only where bf16 rows run).
    cudaError_t linear(bool few_rows, const skn_tensor *w, int M, const float *in32, int64_t ld32, const __nv_bfloat16 *in16, int64_t ld16,
                       const float *gain, const skn_epi &epi);
    cudaError_t launch_linear(bool few_rows, const skn_linear &l);
    int32_t record_layer(int M);                        // after a layer run, while tracing
    int32_t head(int n, const int32_t *rows);           // logits of n rows of x (rows: device list, NULL for the first n)
};
enum skn_decoder_kind { SKN_KIND_LUGASUN = 1, SKN_KIND_TUTEZEN = 2 };

static inline bool skn_decoder_ok(const skn_decoder *m) { return m && m->magic == SKN_MAGIC_DECODER && skn_ctx_ok(m->ctx); }

struct skn_decoder_sizes {
    int32_t n_layers, width, vocab, loop_start, loop_stop, loop_times, max_seqs, max_tokens, max_ctx, dtype;
    float eps;
};
int32_t skn_decoder_check(skn_ctx *ctx, const skn_decoder_sizes &s);
// fields and run order (no allocation); then, once the model knows its rotations, the buffers
void skn_decoder_init(skn_decoder *m, int kind, skn_ctx *ctx, const skn_decoder_sizes &s);
cudaError_t skn_decoder_allocate(skn_decoder *m);

skn_epi skn_to_rows(int kind, float *y32, int64_t ld32, __nv_bfloat16 *y16, int64_t ld16);
bool skn_dense_is(const skn_tensor *t, const skn_ctx *ctx, int64_t rows, int64_t cols);
// a weight row and one activation row in the matvec kernel's shared memory
static inline bool skn_fits_matvec(const skn_tensor *t) { return !t || t->pitch <= 64 * 1024; }
int32_t skn_put_floats(skn_ctx *ctx, float *dst, const float *host, size_t n);
