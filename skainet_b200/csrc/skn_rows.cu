// Row-wise kernels around the dense linear layers: embedding rows, RMS norms (with an optional normalised addend
// that joins the residual stream first), conversions, and the token side input of a few rows in one launch.
#include "skn_dense.cuh"
#include "skn_ptx.cuh"

#include <cooperative_groups.h>
namespace cg = cooperative_groups;

__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xFFFF0000u); }

__device__ __forceinline__ float row_block_sum(float v, float *red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (int w = 0; w < (int)(blockDim.x >> 5); ++w) t += red[w];
    __syncthreads();
    return t;
}

__global__ void __launch_bounds__(256)
skn_embed_bf16_kernel(const uint8_t *__restrict__ table, int64_t pitch, int64_t n_rows, int D, const int32_t *ids, float *out, float *out2, int64_t ld) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    int64_t id = ids[blockIdx.x];
    if (id < 0 || id >= n_rows) id = 0;            // out-of-range ids read row 0 (no fault)
    const __nv_bfloat16 *src = reinterpret_cast<const __nv_bfloat16 *>(table + id * pitch);
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        const float v = __bfloat162float(src[i]);
        out[blockIdx.x * ld + i] = v;
        if (out2) out2[blockIdx.x * ld + i] = v;
    }
}

cudaError_t skn_launch_embed_bf16(const skn_tensor *table, const int32_t *ids, int M, float *out, float *out2, int64_t ld, cudaStream_t st) {
    if (M == 0) return cudaSuccess;
    return skn_launch_pdl(skn_embed_bf16_kernel, dim3(M), dim3(256), 0, st, 1, (const uint8_t *)table->d_blocks, table->pitch, table->n_rows,
                          (int)table->n_cols, ids, out, out2, ld);
}

// one CTA per row
__global__ void __launch_bounds__(256)
skn_norm_rows_kernel(float *x, int64_t ldx, int D, float eps, const float *add, int64_t ld_add, const float *__restrict__ add_gain,
                     const float *__restrict__ gain, skn_rows_out out, __nv_bfloat16 *raw16, int64_t ld_raw16, const int32_t *rows) {
    __shared__ float red[8];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int64_t m = blockIdx.x, src = rows ? rows[m] : m;
    float *xr = x + src * ldx;
    if (add) {
        const float *ar = add + m * ld_add;
        float ss = 0.f;
        for (int i = threadIdx.x; i < D; i += 256) ss = fmaf(ar[i], ar[i], ss);
        const float r = 1.f / sqrtf(row_block_sum(ss, red) / (float)D + eps);
        for (int i = threadIdx.x; i < D; i += 256) xr[i] += ar[i] * r * add_gain[i];      // a thread re-reads its own columns below
    }
    if (raw16)
        for (int i = threadIdx.x; i < D; i += 256) raw16[m * ld_raw16 + i] = __float2bfloat16_rn(xr[i]);
    if (!gain) return;
    float ss = 0.f;
    for (int i = threadIdx.x; i < D; i += 256) ss = fmaf(xr[i], xr[i], ss);
    const float r = 1.f / sqrtf(row_block_sum(ss, red) / (float)D + eps);
    for (int i = threadIdx.x; i < D; i += 256) {
        const float v = xr[i] * r * gain[i];
        if (out.y32) out.y32[m * out.ld32 + i] = v;
        if (out.y16) out.y16[m * out.ld16 + i] = __float2bfloat16_rn(v);
    }
}

// The same for widths that are multiples of four: the row stays in registers, NV vectors per thread.
template <int NV>
__global__ void __launch_bounds__(256)
skn_norm_rows_vec_kernel(float *x, int64_t ldx, int D, float eps, const float *add, int64_t ld_add, const float *__restrict__ add_gain,
                         const float *__restrict__ gain, skn_rows_out out, __nv_bfloat16 *raw16, int64_t ld_raw16, const int32_t *rows) {
    __shared__ float red[8];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int64_t m = blockIdx.x, src = rows ? rows[m] : m;
    float *xr = x + src * ldx;
    float4 v[NV];
#pragma unroll
    for (int u = 0; u < NV; ++u) {
        const int i = (u * 256 + threadIdx.x) * 4;
        v[u] = i < D ? *reinterpret_cast<const float4 *>(xr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (add) {
        float4 a[NV];
        float ss = 0.f;
#pragma unroll
        for (int u = 0; u < NV; ++u) {
            const int i = (u * 256 + threadIdx.x) * 4;
            a[u] = i < D ? *reinterpret_cast<const float4 *>(add + m * ld_add + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            ss += a[u].x * a[u].x + a[u].y * a[u].y + a[u].z * a[u].z + a[u].w * a[u].w;
        }
        const float r = 1.f / sqrtf(row_block_sum(ss, red) / (float)D + eps);
#pragma unroll
        for (int u = 0; u < NV; ++u) {
            const int i = (u * 256 + threadIdx.x) * 4;
            if (i < D) {
                const float4 g = __ldg(reinterpret_cast<const float4 *>(add_gain + i));
                v[u].x += a[u].x * r * g.x; v[u].y += a[u].y * r * g.y; v[u].z += a[u].z * r * g.z; v[u].w += a[u].w * r * g.w;
                *reinterpret_cast<float4 *>(xr + i) = v[u];
            }
        }
    }
    auto put16 = [&](__nv_bfloat16 *p, float4 f) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(f.x, f.y), b = __floats2bfloat162_rn(f.z, f.w);
        uint2 w;
        w.x = *reinterpret_cast<const uint32_t *>(&a);
        w.y = *reinterpret_cast<const uint32_t *>(&b);
        *reinterpret_cast<uint2 *>(p) = w;
    };
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < NV; ++u) {
        const int i = (u * 256 + threadIdx.x) * 4;
        if (raw16 && i < D) put16(raw16 + m * ld_raw16 + i, v[u]);
        ss += v[u].x * v[u].x + v[u].y * v[u].y + v[u].z * v[u].z + v[u].w * v[u].w;
    }
    if (!gain) return;
    const float r = 1.f / sqrtf(row_block_sum(ss, red) / (float)D + eps);
#pragma unroll
    for (int u = 0; u < NV; ++u) {
        const int i = (u * 256 + threadIdx.x) * 4;
        if (i >= D) continue;
        const float4 g = __ldg(reinterpret_cast<const float4 *>(gain + i));
        const float4 f = make_float4(v[u].x * r * g.x, v[u].y * r * g.y, v[u].z * r * g.z, v[u].w * r * g.w);
        if (out.y32) *reinterpret_cast<float4 *>(out.y32 + m * out.ld32 + i) = f;
        if (out.y16) put16(out.y16 + m * out.ld16 + i, f);
    }
}

cudaError_t skn_launch_norm_rows(float *x, int64_t ldx, int M, int D, float eps, const float *add, int64_t ld_add,
                                 const float *add_gain, const float *gain, const skn_rows_out &out, __nv_bfloat16 *raw16,
                                 int64_t ld_raw16, const int32_t *rows, cudaStream_t st) {
    if (M == 0) return cudaSuccess;
    if (D % 4 == 0 && D <= 8192 && ldx % 4 == 0 && ld_add % 4 == 0 && out.ld32 % 4 == 0 && out.ld16 % 4 == 0 && ld_raw16 % 4 == 0) {
#define NORM_CASE(NV) skn_launch_pdl(skn_norm_rows_vec_kernel<NV>, dim3(M), dim3(256), 0, st, 1, x, ldx, D, eps, add, ld_add, add_gain, gain, out, raw16, ld_raw16, rows)
        return D <= 1024 ? NORM_CASE(1) : D <= 2048 ? NORM_CASE(2) : D <= 4096 ? NORM_CASE(4) : NORM_CASE(8);
#undef NORM_CASE
    }
    return skn_launch_pdl(skn_norm_rows_kernel, dim3(M), dim3(256), 0, st, 1, x, ldx, D, eps, add, ld_add, add_gain, gain, out, raw16, ld_raw16, rows);
}

__global__ void __launch_bounds__(256)
skn_concat_bf16_kernel(const float *a, const float *b, int64_t ld, int D, __nv_bfloat16 *out, int64_t ldo) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int64_t m = blockIdx.x;
    for (int i = threadIdx.x; i < D; i += 256) {
        out[m * ldo + i] = __float2bfloat16_rn(a[m * ld + i]);
        if (b) out[m * ldo + D + i] = __float2bfloat16_rn(b[m * ld + i]);
    }
}

cudaError_t skn_launch_concat_bf16(const float *a, const float *b, int64_t ld, int M, int D, __nv_bfloat16 *out, int64_t ldo, cudaStream_t st) {
    if (M == 0) return cudaSuccess;
    return skn_launch_pdl(skn_concat_bf16_kernel, dim3(M), dim3(256), 0, st, 1, a, b, ld, D, out, ldo);
}

cudaError_t skn_launch_rows_to_bf16(const float *in, int64_t ld, int M, int D, __nv_bfloat16 *out, int64_t ldo, cudaStream_t st) {
    return skn_launch_concat_bf16(in, nullptr, ld, M, D, out, ldo, st);
}

// ---- token side input, a few rows -------------------------------------------------------------------------------
// The cluster of 8 CTAs owns one row: CTA r computes the gate rows r, r + 8, ... and shares them through distributed
// shared memory, then its eighth of the projection's rows; the sum of squares meets the same way.
constexpr int SIDE_CLUSTER = 8, SIDE_THREADS = 512;

__device__ __forceinline__ void prefetch_l2(const void *p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

__global__ void __launch_bounds__(SIDE_THREADS)
skn_token_side_kernel(const uint8_t *__restrict__ wg, int64_t pitch_g, const uint8_t *__restrict__ wp, int64_t pitch_p,
                      const uint8_t *__restrict__ table, int64_t pitch_t, int64_t table_rows, int64_t col, const int32_t *ids, float *x,
                      int64_t ldx, int D, int S, const float *__restrict__ gain, float eps) {
    extern __shared__ float sm[];                      // x row (padded to 8), then g [S padded to 8], then y [rows of this CTA]
    __shared__ float red[SIDE_THREADS / 32], part[SIDE_CLUSTER];
    cg::cluster_group cl = cg::this_cluster();
    const int rank = (int)cl.block_rank(), m = blockIdx.x / SIDE_CLUSTER;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int D8 = (int)(pitch_g / 2), S8 = (int)(pitch_p / 2);
    float *xs = sm, *gs = sm + D8, *ys = gs + S8;
    // this CTA's weights are on their way into L2 while the kernel before still runs
    const int per = (D + SIDE_CLUSTER - 1) / SIDE_CLUSTER, n0 = rank * per, n1 = min(D, n0 + per);
    for (int j = rank + SIDE_CLUSTER * warp; j < S; j += SIDE_CLUSTER * (SIDE_THREADS / 32))
        for (int64_t i = (int64_t)lane * 128; i < pitch_g; i += 32 * 128) prefetch_l2(wg + (int64_t)j * pitch_g + i);
    for (int64_t i = n0 * pitch_p + (int64_t)threadIdx.x * 128; i < n1 * pitch_p; i += SIDE_THREADS * 128) prefetch_l2(wp + i);
    skn_pdl_wait();
    float *xr = x + (int64_t)m * ldx;
    for (int i = threadIdx.x; i < D8; i += SIDE_THREADS) xs[i] = i < D ? __ldcg(xr + i) : 0.f;
    for (int i = threadIdx.x; i < S8; i += SIDE_THREADS) gs[i] = 0.f;
    int64_t id = ids[m];
    if (id < 0 || id >= table_rows) id = 0;
    const __nv_bfloat16 *er = reinterpret_cast<const __nv_bfloat16 *>(table + id * pitch_t) + col;
    __syncthreads();
    cl.sync();                                         // every CTA's g is zeroed before a peer writes into it
    for (int j = rank + SIDE_CLUSTER * warp; j < S; j += SIDE_CLUSTER * (SIDE_THREADS / 32)) {
        const uint4 *wr = reinterpret_cast<const uint4 *>(wg + (int64_t)j * pitch_g);
        float a = 0.f;
#pragma unroll 8
        for (int i = lane; i < D8 / 8; i += 32) {
            const uint4 w = __ldg(wr + i);
            const float4 lo = *reinterpret_cast<const float4 *>(xs + i * 8), hi = *reinterpret_cast<const float4 *>(xs + i * 8 + 4);
            a = fmaf(bf_lo(w.x), lo.x, a); a = fmaf(bf_hi(w.x), lo.y, a); a = fmaf(bf_lo(w.y), lo.z, a); a = fmaf(bf_hi(w.y), lo.w, a);
            a = fmaf(bf_lo(w.z), hi.x, a); a = fmaf(bf_hi(w.z), hi.y, a); a = fmaf(bf_lo(w.w), hi.z, a); a = fmaf(bf_hi(w.w), hi.w, a);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
        a = 0.5f * a * (1.f + tanhf(0.7978845608028654f * (a + 0.044715f * a * a * a))) * __bfloat162float(er[j]);
        if (lane < SIDE_CLUSTER) *cl.map_shared_rank(gs + j, lane) = a;
    }
    cl.sync();
    float ss = 0.f;
    for (int n = n0 + threadIdx.x; n < n1; n += SIDE_THREADS) {
        const uint4 *wr = reinterpret_cast<const uint4 *>(wp + (int64_t)n * pitch_p);
        float a = 0.f;
#pragma unroll 8
        for (int i = 0; i < S8 / 8; ++i) {
            const uint4 w = __ldg(wr + i);
            const float4 lo = *reinterpret_cast<const float4 *>(gs + i * 8), hi = *reinterpret_cast<const float4 *>(gs + i * 8 + 4);
            a = fmaf(bf_lo(w.x), lo.x, a); a = fmaf(bf_hi(w.x), lo.y, a); a = fmaf(bf_lo(w.y), lo.z, a); a = fmaf(bf_hi(w.y), lo.w, a);
            a = fmaf(bf_lo(w.z), hi.x, a); a = fmaf(bf_hi(w.z), hi.y, a); a = fmaf(bf_lo(w.w), hi.z, a); a = fmaf(bf_hi(w.w), hi.w, a);
        }
        ys[n - n0] = a;
        ss = fmaf(a, a, ss);
    }
    ss = row_block_sum(ss, red);
    if (threadIdx.x < SIDE_CLUSTER) *cl.map_shared_rank(part + rank, threadIdx.x) = ss;
    cl.sync();
    float t = 0.f;
#pragma unroll
    for (int r = 0; r < SIDE_CLUSTER; ++r) t += part[r];
    const float r = 1.f / sqrtf(t / (float)D + eps);
    for (int n = n0 + threadIdx.x; n < n1; n += SIDE_THREADS) xr[n] = xs[n] + ys[n - n0] * r * gain[n];
}

static size_t side_smem(const skn_tensor *wg, const skn_tensor *wp) {
    return ((size_t)wg->pitch / 2 + wp->pitch / 2 + (wg->n_cols + SIDE_CLUSTER - 1) / SIDE_CLUSTER) * sizeof(float);
}
bool skn_token_side_fits(const skn_tensor *wg, const skn_tensor *wp) { return side_smem(wg, wp) <= 200 * 1024; }

cudaError_t skn_launch_token_side(const skn_tensor *wg, const skn_tensor *wp, const skn_tensor *table, int64_t col, const int32_t *ids,
                                  float *x, int64_t ldx, int M, const float *gain, float eps, cudaStream_t st) {
    if (M == 0) return cudaSuccess;
    const int D = (int)wg->n_cols, S = (int)wg->n_rows;
    if (!skn_token_side_fits(wg, wp)) return cudaErrorNotSupported;
    const size_t smem = side_smem(wg, wp);
    const cudaError_t e = cudaFuncSetAttribute(skn_token_side_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return e;
    return skn_launch_pdl(skn_token_side_kernel, dim3(M * SIDE_CLUSTER), dim3(SIDE_THREADS), smem, st, SIDE_CLUSTER, (const uint8_t *)wg->d_blocks,
                          wg->pitch, (const uint8_t *)wp->d_blocks, wp->pitch, (const uint8_t *)table->d_blocks, table->pitch, table->n_rows, col, ids, x,
                          ldx, D, S, gain, eps);
}

// ---- norms of parts of a row, vectors added to rows ----------------------------------------------------------------
// A row holds heads of `pitch` columns, the first `head` of each valid; the valid columns, heads in a row, fall into equal parts.
__global__ void __launch_bounds__(256)
skn_part_norm_kernel(const float *x, int64_t ldx, int heads, int head, int pitch, int parts, float eps, const float *__restrict__ gain, skn_rows_out out) {
    __shared__ float red[8];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int64_t m = blockIdx.x;
    const float *xr = x + m * ldx;
    const int len = heads * head / parts, p = blockIdx.y;
    if (head == pitch && len % 4 == 0 && len <= 8192 && ldx % 4 == 0) {
        // the part stays in registers
        float4 v[8];
        float ss = 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int i = (u * 256 + threadIdx.x) * 4;
            v[u] = i < len ? *reinterpret_cast<const float4 *>(xr + p * len + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            ss += v[u].x * v[u].x + v[u].y * v[u].y + v[u].z * v[u].z + v[u].w * v[u].w;
        }
        const float r = 1.f / sqrtf(row_block_sum(ss, red) / (float)len + eps);
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int i = (u * 256 + threadIdx.x) * 4, c = p * len + i;
            if (i >= len) continue;
            const float4 g = __ldg(reinterpret_cast<const float4 *>(gain + c));
            const float4 f = make_float4(v[u].x * r * g.x, v[u].y * r * g.y, v[u].z * r * g.z, v[u].w * r * g.w);
            if (out.y32) {
                float *y = out.y32 + m * out.ld32 + c;
                y[0] = f.x; y[1] = f.y; y[2] = f.z; y[3] = f.w;
            }
            if (out.y16) {
                __nv_bfloat16 *y = out.y16 + m * out.ld16 + c;
                *reinterpret_cast<__nv_bfloat162 *>(y) = __floats2bfloat162_rn(f.x, f.y);
                *reinterpret_cast<__nv_bfloat162 *>(y + 2) = __floats2bfloat162_rn(f.z, f.w);
            }
        }
        return;
    }
    auto column = [&](int i) { return (p * len + i) / head * pitch + (p * len + i) % head; };
    float ss = 0.f;
    for (int i = threadIdx.x; i < len; i += 256) {
        const float v = xr[column(i)];
        ss = fmaf(v, v, ss);
    }
    const float r = 1.f / sqrtf(row_block_sum(ss, red) / (float)len + eps);
    for (int i = threadIdx.x; i < len; i += 256) {
        const int c = column(i);
        const float v = xr[c] * r * gain[c];
        if (out.y32) out.y32[m * out.ld32 + c] = v;
        if (out.y16) out.y16[m * out.ld16 + c] = __float2bfloat16_rn(v);
    }
}

cudaError_t skn_launch_part_norm_rows(const float *x, int64_t ldx, int M, int heads, int head, int pitch, int parts, float eps, const float *gain,
                                      const skn_rows_out &out, cudaStream_t st) {
    if (M == 0) return cudaSuccess;
    return skn_launch_pdl(skn_part_norm_kernel, dim3(M, parts), dim3(256), 0, st, 1, x, ldx, heads, head, pitch, parts, eps, gain, out);
}

__global__ void __launch_bounds__(256)
skn_add_vec_rows_kernel(float *x, int64_t ldx, int D, const float *__restrict__ vec, const float *add, int64_t ld_add) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int64_t m = blockIdx.x;
    for (int i = threadIdx.x; i < D; i += 256) {
        float v = x[m * ldx + i];
        if (add) v += add[m * ld_add + i];
        x[m * ldx + i] = v + vec[i];
    }
}

cudaError_t skn_launch_add_vec_rows(float *x, int64_t ldx, int M, int D, const float *vec, const float *add, int64_t ld_add, cudaStream_t st) {
    if (M == 0) return cudaSuccess;
    return skn_launch_pdl(skn_add_vec_rows_kernel, dim3(M), dim3(256), 0, st, 1, x, ldx, D, vec, add, ld_add);
}
