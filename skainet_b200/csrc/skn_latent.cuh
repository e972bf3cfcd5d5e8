// Latent attention (declarations; kernels in skn_latent.cu): queries and keys / values go through normalised latents, and the cache holds one
// row per token, [latent | rotated key part shared by the heads], in a position-addressed cache of one key head without V.
//   absorbed   a query meets the latents themselves: q~ = W_uk^T q, scores q~ . c + q_rot . k_rot, the weighted latent then goes through W_uv.
//              Serves single tokens, short portions and the fp32 decoder
//   expanded   keys and values of every head are formed from the cached latents once per step and the tile kernel runs over them.
//              Serves many tokens
// Widths dim, vdim and kvp (the latent's) are multiples of 8, dim + rp of 16; padding is zero.  Adjacent dimensions of the rotated part
// form the pairs.
#pragma once
#include "skn_mixers.cuh"
#include "skn_moe.cuh"

struct skn_latent_args {
    const skn_kvcache *kv;          // k_dim = kvp + rp
    int heads, dim, rp, vdim, q_rank, kv_rank, kvp, window;
    float scale, eps;
    const float *q_gain, *kv_gain, *sink;
    skn_rot rot;
    const float *dq, *dkv, *gate;   // raw parts of the joint row of token 0: [q_rank], [kvp | rp], [heads][vdim]; rows are ld apart
    int64_t ld;
    const skn_tensor *uq, *ukv;
    skn_rows_out out;
    skn_route_args route;           // rides along in the absorbed form's first launch
    float *q;                       // [rows][heads][dim + rp], before rotation
    float *ql, *ol;                 // absorbed: [rows][heads][kvp + rp], [rows][heads][kvp]
    float *scratch;                 // skn_latent_scratch() floats
    unsigned *tickets;
    float *cq32;                    // normalised query latents, [rows][q_rank rounded up to 8]
    __nv_bfloat16 *cq16;
    __nv_bfloat16 *q16;             // expanded: [rows][heads][dim + rp], rotated
    __nv_bfloat16 *kvx;             // expanded: [ring slots][heads * (dim + vdim)]
};

// floats of scratch for the absorbed form of up to `rows` rows
size_t skn_latent_scratch(const skn_latent_args &a, int rows, int max_pos);
bool skn_latent_expand_fits(const skn_latent_args &a);
// The newest latents and rotated keys into the cache, and the normalised query latents to cq (either form, where given)
cudaError_t skn_launch_latent_rows(const skn_step &s, const skn_latent_args &a, const skn_rows_out &cq, cudaStream_t st);
// Absorbed form, from a.q on (three launches); append: the first one also files the newest latents
cudaError_t skn_launch_latent_absorbed(const skn_step &s, const skn_latent_args &a, bool append, cudaStream_t st);
// Expanded form, from a.q16 on: one sequence of the step at a time, len[i] tokens of sequence i being in the cache by now
cudaError_t skn_launch_latent_expanded(skn_ctx *ctx, const skn_step &s, const skn_latent_args &a, const int32_t *len, const skn_dense_ws &ws, cudaStream_t st);
int32_t skn_check_latent_spec(skn_ctx *ctx, const skn_latent_spec *s);
