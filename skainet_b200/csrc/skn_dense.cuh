// Linear layers over dense bf16 weights, with what surrounds them in a decoder folded in (declarations; the kernels
// are in skn_dense.cu), and the row-wise kernels that feed them (skn_rows.cu).
#pragma once
#include "skn_internal.cuh"
#include <cuda_bf16.h>

// what happens to acc = W[n] . x[m] before it is stored
enum skn_epi_kind {
    SKN_EPI_STORE = 0,      // acc
    SKN_EPI_ADD = 1,        // resid[m][n] + alpha * acc
    SKN_EPI_RELU2 = 2,      // max(acc, 0)^2
    SKN_EPI_GELU_TABLE = 3, // gelu_tanh(acc) * table[ids[m]][table_col + n]
    // several layers that read the same x, stacked: rows below n_act go to y32 as they are, the others to act*
    SKN_EPI_GELU_TAIL = 4,  // gelu_tanh(acc), column n - n_act
    SKN_EPI_SILU_TAIL = 5,  // rows in pairs (gate, up), n_act even: silu(gate) * up, column (n - n_act) / 2
    SKN_EPI_ROTATE = 6      // rows in heads of rot_head: adjacent pairs from dimension rot_lo on turn by the row's angles
};
__host__ __device__ constexpr bool skn_epi_pairs(int kind) { return kind == SKN_EPI_SILU_TAIL || kind == SKN_EPI_ROTATE; }

struct skn_rot {                    // angles of a step: row m, pair i at table[m * ld + i] = (cos, sin); half = 0: no rotation
    const float2 *table;
    int ld, half;
};

struct skn_epi {
    int kind;
    float alpha;                        // SKN_EPI_ADD
    const float *resid;                 // SKN_EPI_ADD; may alias y32
    int64_t ld_resid;
    const __nv_bfloat16 *table;         // SKN_EPI_GELU_TABLE
    int64_t ld_table, table_rows, table_col;
    const int32_t *ids;
    int n_act;                          // SKN_EPI_*_TAIL: either or both outputs
    float *act32;
    int64_t ld_act32;
    __nv_bfloat16 *act16;
    int64_t ld_act16;
    const float *act_scale;             // SKN_EPI_SILU_TAIL: optional factor act_scale[(n - n_act) / scale_rows]
    int scale_rows;
    skn_rot rot;                        // SKN_EPI_ROTATE
    int rot_head, rot_lo;
    float *y32;                         // either or both outputs
    int64_t ld_y32;
    __nv_bfloat16 *y16;
    int64_t ld_y16;
};

// How a linear layer picks among stacked experts on the device.
enum skn_pick_kind {
    SKN_PICK_NONE = 0,
    SKN_PICK_ROWS = 1,                  // matvec: the weight rows of experts expert[0 .. n - 1] (rows_per each), one after the other
    SKN_PICK_COLS = 2,                  // matvec: row n is [w row n | row n of expert[0] of w2 | row n of expert[1] ..]
    SKN_PICK_GROUPS = 3                 // many rows: rows offset[e] .. offset[e + 1] - 1 of x meet expert e (rows_per rows of w)
};
struct skn_pick {
    int kind, n;                        // n: experts picked (matvec), all experts (groups)
    const int32_t *expert;              // device
    const skn_tensor *w2;               // SKN_PICK_COLS: [experts * rows][columns]
    int rows_per;
    const int32_t *offset;              // device, [n + 1]; SKN_PICK_GROUPS
};
constexpr int SKN_MAX_EXPERTS = 1024;

struct skn_linear {
    const skn_tensor *w;                // SKN_TYPE_BF16
    int M;
    const float *x32;                   // fp32 rows (matvec and fp32 kernels) ...
    int64_t ld_x32;
    const float *x32b;                  // ... optionally continued by a second matrix: K = k_a columns of x32, the rest of x32b
    int64_t ld_x32b, k_a;
    const float *gain;                  // ... optionally RMS-normalised first: x / sqrt(mean(x^2) + eps) * gain (matvec kernel only),
    int norm_cols, norm_parts;          //     norm_cols > 0: only the first norm_cols columns, in equal parts (widths multiples of 8)
    float eps;
    const __nv_bfloat16 *x16;           // bf16 rows (tensor-core kernel); pitch in elements, a multiple of 8
    int64_t ld_x16;
    skn_pick pick;
    skn_epi epi;
};
// columns of the joint weight row: w's, and w2's for every picked expert
static inline int64_t skn_linear_cols(const skn_linear &l) {
    return l.pick.kind == SKN_PICK_COLS ? l.w->pitch / 2 + l.pick.n * (l.pick.w2->pitch / 2) : l.w->n_cols;
}

// rows a linear layer takes on the matvec kernel (fp32 x, weights streamed once, norm folded in)
constexpr int SKN_MATVEC_ROWS = 4;

// split-K workspace of the tensor-core kernel
constexpr int SKN_DENSE_MAX_TILES = 2048;
struct skn_dense_ws {
    float *partial;                     // SKN_DENSE_WS_FLOATS
    unsigned *tickets;                  // SKN_DENSE_MAX_TILES, zero between launches
};
constexpr size_t SKN_DENSE_WS_FLOATS = (size_t)8 << 20;

// most parts of a partial norm, and whether the matvec kernel takes such a norm
constexpr int SKN_NORM_PARTS = 16;
static inline bool skn_norm_folds(int cols, int parts) { return parts <= SKN_NORM_PARTS && cols % parts == 0 && cols / parts % 8 == 0; }
// matvec kernel (M <= SKN_MATVEC_ROWS; more rows are served by several launches; picks: M = 1)
cudaError_t skn_launch_dense_matvec(skn_ctx *ctx, const skn_linear &l, cudaStream_t st);
// plain fp32 products of fp32 rows, any M
cudaError_t skn_launch_dense_f32(skn_ctx *ctx, const skn_linear &l, cudaStream_t st);
// tensor cores: bf16 rows, fp32 accumulation, any M
cudaError_t skn_launch_dense_tc(skn_ctx *ctx, const skn_linear &l, const skn_dense_ws &ws, cudaStream_t st);

// ---- row-wise kernels (skn_rows.cu) ---------------------------------------------------------------------
// A destination of fp32 and / or bf16 rows.
struct skn_rows_out {
    float *y32;
    int64_t ld32;
    __nv_bfloat16 *y16;
    int64_t ld16;
};
// out[m] = table[ids[m]] (fp32), to one or two destinations
cudaError_t skn_launch_embed_bf16(const skn_tensor *table, const int32_t *ids, int M, float *out, float *out2, int64_t ld, cudaStream_t st);
// One pass over the rows of the residual stream:
//   add != NULL:  x[m] += add[m] / sqrt(mean(add[m]^2) + eps) * add_gain     (written back)
//   raw.y*:       x[m] as it then is (raw.y32 unused)
//   gain != NULL: out = x[m] / sqrt(mean(x[m]^2) + eps) * gain
// rows: optional list of source rows (gather).
cudaError_t skn_launch_norm_rows(float *x, int64_t ldx, int M, int D, float eps, const float *add, int64_t ld_add,
                                 const float *add_gain, const float *gain, const skn_rows_out &out, __nv_bfloat16 *raw16,
                                 int64_t ld_raw16, const int32_t *rows, cudaStream_t st);
// rows of D columns in heads of `head` valid of `pitch` columns: `parts` equal parts of the valid columns each divided by their own root mean
// square, times gain (padded like x).  out may alias x.
cudaError_t skn_launch_part_norm_rows(const float *x, int64_t ldx, int M, int heads, int head, int pitch, int parts, float eps, const float *gain,
                                      const skn_rows_out &out, cudaStream_t st);
// x[m] += vec (+ add[m] when given)
cudaError_t skn_launch_add_vec_rows(float *x, int64_t ldx, int M, int D, const float *vec, const float *add, int64_t ld_add, cudaStream_t st);
// out16[m] = in[m]
cudaError_t skn_launch_rows_to_bf16(const float *in, int64_t ld, int M, int D, __nv_bfloat16 *out, int64_t ldo, cudaStream_t st);
// out16[m] = [a[m] | b[m]]
cudaError_t skn_launch_concat_bf16(const float *a, const float *b, int64_t ld, int M, int D, __nv_bfloat16 *out, int64_t ldo, cudaStream_t st);
// Token side input of a few rows in one launch (a cluster of 8 CTAs per row):
//   g = gelu_tanh(Wg x) * table[id][col ..], y = Wp g, x += y / sqrt(mean(y^2) + eps) * gain
bool skn_token_side_fits(const skn_tensor *wg, const skn_tensor *wp);
cudaError_t skn_launch_token_side(const skn_tensor *wg, const skn_tensor *wp, const skn_tensor *table, int64_t col, const int32_t *ids,
                                  float *x, int64_t ldx, int M, const float *gain, float eps, cudaStream_t st);

// launch with programmatic stream serialisation: the kernel must call skn_pdl_wait() in every thread before it
// touches anything a kernel before it in the stream wrote
template <class... KArgs, class... Args>
static inline cudaError_t skn_launch_pdl(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, int cluster, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    int n = 0;
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n++].val.programmaticStreamSerializationAllowed = skn_tune_int("SKN_PDL", 1);
    if (cluster > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = cluster;
        attr[n].val.clusterDim.y = 1;
        attr[n++].val.clusterDim.z = 1;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    return cudaLaunchKernelEx(&cfg, kern, args...);
}
