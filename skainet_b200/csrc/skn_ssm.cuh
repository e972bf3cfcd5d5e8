// Selective state space (declarations; kernels in skn_ssm.cu): per head S <- exp(a dt) S + dt B x^T, y = S^T C + D x, where a = -exp(A_log), x, B
// and C come out of a causal convolution per channel with silu, dt = softplus(raw + bias), and y is multiplied by silu(z).
// Head width vp and state width np are multiples of 8 (zero-padded); a joint row is
//     z [heads][vp] | x [heads][vp] | B [groups][np] | C [groups][np] | dt [heads]
// and the convolution's channels are x | B | C.  Its last inputs live in a ring of `taps` rows per sequence (position p in row p % taps),
// one more than it looks back on, so the row that a token fills is none of those it reads.
#pragma once
#include "skn_mixers.cuh"
#include "skn_moe.cuh"

constexpr int SKN_SSM_CHUNK = 64;

struct skn_ssm_args {
    const skn_state *state;             // [heads][np][vp]
    const skn_state *ring;              // [1][taps][channels]
    int heads, vp, np, groups, taps;
    const float *conv, *conv_b;         // [taps][channels], [channels]
    const float *dt_bias, *a, *d;       // [heads]
    const float *proj;                  // joint row of token 0; rows are ld apart
    int64_t ld;
    float *y;                           // gated rows [heads][vp], ld_y apart
    int64_t ld_y;
    skn_route_args route;               // rides along in the step kernel
    // many-token form
    __nv_bfloat16 *xbc;                 // [rows][channels]
    float *dt, *cum;                    // [rows][heads]: step sizes, and the log decays summed from the chunk's start
    float *chunks;                      // what each chunk adds to the state: [seqs][chunks][heads][np][vp]
    __nv_bfloat16 *starts;              // the states at the chunk starts: [seqs][chunks][heads][2 terms][np][vp]
};
__host__ __device__ static inline int skn_ssm_channels(int heads, int vp, int groups, int np) { return heads * vp + 2 * groups * np; }

// tokens one by one, fp32 throughout, any T (one launch; a second one files the convolution's inputs when T > 1)
cudaError_t skn_launch_ssm_step(const skn_step &s, const skn_ssm_args &a, cudaStream_t st);
// chunks of SKN_SSM_CHUNK tokens on the tensor cores
bool skn_ssm_chunks_fit(int vp, int np);
cudaError_t skn_launch_ssm_chunks(const skn_step &s, const skn_ssm_args &a, cudaStream_t st);
int32_t skn_check_ssm_spec(skn_ctx *ctx, const skn_ssm_spec *s);
