// Token mixers over position-addressed caches and recurrent states (declarations; kernels in skn_mixers.cu):
//   attention           per-head RMS norm of q and k, rotation of their first dimensions (half-split pairs), softmax
//                       over the keys of the query's own chunk, of a sliding window, or all earlier keys, optional tanh
//                       soft cap, optional sink in the denominator
//   retention           linear attention with one fixed decay per head: S <- decay S + k v^T, o = S^T q; o divided by
//                       its root mean square and multiplied by silu(gate)
// Both read the raw fp32 rows of one joint projection and write the (scaled) concatenated heads that the output
// projection takes.  Rows are [seq][t], sequence s of a step is slot slot0 + s, and pos[slot] tokens came before.
#pragma once
#include "skn_dense.cuh"

struct skn_step {
    int slot0, n_seqs, T;
    const int32_t *pos;             // device, per slot
    int max_pos;                    // positions are below this
};

struct skn_attn_args {
    const skn_kvcache *kv;
    int heads;
    int chunk, window;              // 0: every earlier key is visible; else the query's chunk, or the last `window` positions
    const float *sink;              // [heads] scores that join the softmax denominator, NULL: none
    float scale, softcap;           // softcap 0: none
    float eps;
    const float *q_gain, *k_gain;   // [dim], NULL: no norm
    skn_rot rot;
    const float *q, *k, *v;         // raw heads of row 0; rows are ld apart
    int64_t ld;
    float out_scale;
    skn_rows_out out;               // pointers at the first column of this mixer's heads
    const float *gate;              // raw gate rows [heads][vdim] whose sigmoid multiplies the heads (tile kernel only), NULL: none
    int64_t ld_gate;
    float *scratch;                 // skn_attn_scratch() floats
    unsigned *tickets;              // rows * heads, zero between launches
    __nv_bfloat16 *q16;             // [rows][heads][k_pitch] (tensor-core form)
};

// Where the tile kernel finds keys and values (bf16).  Slot s of the ring of sequence b, key head g: the first k1 elements of a key at
// k + b k_slot + g k_head + s k_row, the rest (shared by the heads) at k2 + b k2_slot + s k2_row.  Every stride and width is a multiple of
// 8 elements, kp of 16.
struct skn_attn_keys {
    const __nv_bfloat16 *k, *k2, *v;
    int64_t k_row, k_head, k_slot, k2_row, k2_slot, v_row, v_head, v_slot;
    int k1, kp, vp, vdim, cap, group;   // group: query heads per key head
};

struct skn_ret_args {
    const skn_state *state;
    float eps;
    skn_rot rot;
    float k_scale;
    const float *powers;            // [heads][SKN_RET_CHUNK + 1]: decay^n
    float *q, *k;                   // raw heads of row 0 (rotated in place by the many-token form)
    const float *v, *g;
    int64_t ld;
    float out_scale;
    skn_rows_out out;
    bool exact;                     // fp32 products only (no tensor cores)
    float *chunks;                  // [n_seqs][ceil(T / SKN_RET_CHUNK)][heads][k_dim][v_pitch] floats
};
constexpr int SKN_RET_CHUNK = 64;
constexpr int SKN_ATTN_SPLIT_KEYS = 128;

// most key splits a query can need; span: chunk or window, 0 for none
static inline int skn_attn_splits(int span, int max_pos) {
    const int n = span > 0 && span < max_pos ? span : max_pos;
    return (n + SKN_ATTN_SPLIT_KEYS - 1) / SKN_ATTN_SPLIT_KEYS;
}
// floats of scratch for `rows` query rows on the split kernel
static inline size_t skn_attn_scratch(int rows, int heads, int v_dim, int span, int max_pos) {
    const int s = skn_attn_splits(span, max_pos);
    return s > 1 ? (size_t)rows * heads * s * (v_dim + 2) : 1;
}
// whether many-token steps of this cache run on the tensor-core kernel (bf16 cache, head widths up to 256)
bool skn_chunk_attn_tc(const skn_kvcache *kv);

bool skn_attn_tiles_fit(int kp, int vp);
// attention of prepared queries over the cache, whose newest keys are in place: any element type, any number of tokens
cudaError_t skn_launch_attn_rows(const skn_step &s, const skn_attn_args &a, cudaStream_t st);
// the same on the tensor-core tile kernel, queries in a.q16
cudaError_t skn_launch_attn_tiles(const skn_step &s, const skn_attn_args &a, const skn_attn_keys &k, cudaStream_t st);

// (cos, sin) of pos * freq[i] for every row of the step; angles in double
cudaError_t skn_launch_rot_table(const skn_step &s, const double *freq, int half, float2 *out, int ld, cudaStream_t st);
// single-token step: norm, rotation, cache append, attention and state update in one launch; either part may be NULL
cudaError_t skn_launch_mix_decode(skn_ctx *ctx, const skn_step &s, const skn_attn_args *a, const skn_ret_args *r, cudaStream_t st);
// many-token step: heads prepared and appended by one launch, then attention, then retention in chunks
cudaError_t skn_launch_mix_prefill(skn_ctx *ctx, const skn_step &s, const skn_attn_args *a, const skn_ret_args *r, cudaStream_t st);
// pos[slot0 + s] += T (a length that would pass max_pos stays there and SKN_ERR_SHAPE lands in the status word)
cudaError_t skn_launch_advance(const skn_step &s, int32_t *pos, int32_t *status, cudaStream_t st);

// host side: rotation frequencies base^(-2 i / dims), decay powers [heads][SKN_RET_CHUNK + 1], and checks of the public specs
void skn_rot_freqs(double base, int dims, double *out);
void skn_decay_powers(const double *decay, int heads, float *out);
int32_t skn_check_attn_spec(skn_ctx *ctx, const skn_attn_spec *a);
int32_t skn_check_retention_spec(skn_ctx *ctx, const skn_retention_spec *r);
