// Mixture-of-experts routing and the row movement around the experts' linear layers (kernels in skn_moe.cu).
//   few rows     the choice of a row rides in the mixer's launch (skn_route_row); the matvec kernel then picks the experts' weights
//   many rows    choice, grouping of the (token, choice) pairs by expert, rows gathered in that order, two grouped linear layers,
//                and the weighted sum of each token's expert outputs
#pragma once
#include "skn_dense.cuh"

struct skn_route_args {
    const float *logits;            // row 0's router logits; rows are ld apart.  NULL: nothing to route
    int64_t ld;
    int experts, top;
    int32_t *expert;                // [rows][top], best first
    float *weight;                  // [rows][top]: softmax scores of the chosen, divided by their sum + 1e-20
};
static inline size_t skn_route_smem(const skn_route_args &r) { return r.logits ? (size_t)r.experts * sizeof(float) : 0; }

#ifdef __CUDACC__
// One warp: the `top` largest of the row's softmax scores (ties: the lower index).  z: `experts` floats of shared memory.
__device__ __forceinline__ void skn_route_row(const skn_route_args &r, int64_t m, float *z) {
    const int lane = threadIdx.x & 31;
    float mx = -INFINITY;
    for (int e = lane; e < r.experts; e += 32) {
        const float v = __ldcg(r.logits + m * r.ld + e);
        z[e] = v;
        mx = fmaxf(mx, v);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.f;
    for (int e = lane; e < r.experts; e += 32) {
        z[e] = expf(z[e] - mx);
        sum += z[e];
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    __syncwarp();
    float total = 0.f;
    for (int k = 0; k < r.top; ++k) {
        float best = -1.f;          // taken entries hold -2, so an index in range is found whatever the values are
        int at = r.experts;
        for (int e = lane; e < r.experts; e += 32) {
            const float v = z[e];
            if (v != -2.f && (v > best || at == r.experts)) {
                best = v;
                at = e;
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float v = __shfl_xor_sync(0xffffffffu, best, o);
            const int i = __shfl_xor_sync(0xffffffffu, at, o);
            if (i < r.experts && (at == r.experts || v > best || (v == best && i < at))) {
                best = v;
                at = i;
            }
        }
        at = __shfl_sync(0xffffffffu, at, 0);
        if (at >= r.experts) at = 0;
        const float s = z[at] / sum;
        total += s;
        __syncwarp();
        if (lane == 0) {
            r.expert[m * r.top + k] = at;
            r.weight[m * r.top + k] = s;
            z[at] = -2.f;
        }
        __syncwarp();
    }
    for (int k = lane; k < r.top; k += 32) {
        // written by lane 0 above; the warp is in step and the stores are visible to it after the barrier
        float *w = r.weight + m * r.top + k;
        *w = *reinterpret_cast<volatile float *>(w) / (total + 1e-20f);
    }
}
#endif

// choice of every row
cudaError_t skn_launch_route(const skn_route_args &r, int M, cudaStream_t st);
// pairs i = m * top + k grouped by expert, in order of i: offset[experts + 1], and place[i], the pair's row in the grouped order
cudaError_t skn_launch_group_pairs(const int32_t *expert, int pairs, int experts, int32_t *offset, int32_t *place, cudaStream_t st);
// row place[m * top + k] of the grouped rows = row m (bf16 or fp32, whichever is given), k < top
cudaError_t skn_launch_scatter_rows(const skn_rows_out &rows, int M, int D, int top, const int32_t *place, const skn_rows_out &out, cudaStream_t st);
// x[m] += alpha * sum over k of weight[m][k] * y[place[m * top + k]]
cudaError_t skn_launch_gather_experts(float *x, int64_t ldx, int M, int D, float alpha, int top, const int32_t *place, const float *weight,
                                      const skn_rows_out &y, cudaStream_t st);
