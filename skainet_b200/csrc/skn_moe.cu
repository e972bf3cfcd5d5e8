// Routing and row movement of the mixture of experts (see skn_moe.cuh).
#include "skn_moe.cuh"
#include "skn_ptx.cuh"

__global__ void __launch_bounds__(32)
skn_route_kernel(skn_route_args r) {
    extern __shared__ float z[];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    skn_route_row(r, blockIdx.x, z);
}

cudaError_t skn_launch_route(const skn_route_args &r, int M, cudaStream_t st) {
    return skn_launch_pdl(skn_route_kernel, dim3(M), dim3(32), skn_route_smem(r), st, 1, r);
}

constexpr int GP_THREADS = 1024;

// CTA e reads every pair: those of lower experts count towards its offset, its own get consecutive places
__global__ void __launch_bounds__(GP_THREADS)
skn_group_pairs_kernel(const int32_t *expert, int pairs, int experts, int32_t *offset, int32_t *place) {
    __shared__ int below[GP_THREADS], own[GP_THREADS], base_s;
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int e = blockIdx.x, tid = threadIdx.x, per = (pairs + GP_THREADS - 1) / GP_THREADS, i0 = min(pairs, tid * per), i1 = min(pairs, i0 + per);
    int lo = 0, eq = 0;
#pragma unroll 8
    for (int i = i0; i < i1; ++i) {
        const int v = __ldcg(expert + i);
        lo += v < e;
        eq += v == e;
    }
    below[tid] = lo;
    own[tid] = eq;
    __syncthreads();
    if (tid < 32) {
        int total = 0, run = 0;
        for (int j = 0; j < GP_THREADS / 32; ++j) {
            total += below[tid * (GP_THREADS / 32) + j];
            run += own[tid * (GP_THREADS / 32) + j];
        }
        int before = run;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int y = __shfl_up_sync(0xffffffffu, before, o);
            if (tid >= o) before += y;
        }
        before -= run;
        for (int j = 0; j < GP_THREADS / 32; ++j) {
            const int n = own[tid * (GP_THREADS / 32) + j];
            own[tid * (GP_THREADS / 32) + j] = before;
            before += n;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) total += __shfl_xor_sync(0xffffffffu, total, o);
        if (tid == 0) {
            base_s = total;
            offset[e] = total;
            if (e == experts - 1) offset[experts] = pairs;
        }
    }
    __syncthreads();
    int at = base_s + own[tid];
#pragma unroll 8
    for (int i = i0; i < i1; ++i)
        if (__ldcg(expert + i) == e) place[i] = at++;
}

cudaError_t skn_launch_group_pairs(const int32_t *expert, int pairs, int experts, int32_t *offset, int32_t *place, cudaStream_t st) {
    return skn_launch_pdl(skn_group_pairs_kernel, dim3(experts), dim3(GP_THREADS), 0, st, 1, expert, pairs, experts, offset, place);
}

// rows in 16-byte pieces (pitches are multiples of 8 elements, padding included)
__global__ void __launch_bounds__(256)
skn_scatter_rows_kernel(const uint4 *rows, int64_t ld, int n, int top, const int32_t *place, uint4 *out, int64_t ldo) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int64_t m = blockIdx.x;
    for (int i = threadIdx.x; i < n; i += 256) {
        const uint4 v = rows[m * ld + i];
        for (int k = 0; k < top; ++k) out[place[m * top + k] * ldo + i] = v;
    }
}

cudaError_t skn_launch_scatter_rows(const skn_rows_out &rows, int M, int D, int top, const int32_t *place, const skn_rows_out &out, cudaStream_t st) {
    const int es = rows.y32 ? 4 : 2;
    const int64_t ld = (rows.y32 ? rows.ld32 : rows.ld16) * es, ldo = (rows.y32 ? out.ld32 : out.ld16) * es;
    if (ld % 16 || ldo % 16) return cudaErrorInvalidValue;
    const void *src = rows.y32 ? (const void *)rows.y32 : rows.y16;
    void *dst = rows.y32 ? (void *)out.y32 : out.y16;
    return skn_launch_pdl(skn_scatter_rows_kernel, dim3(M), dim3(256), 0, st, 1, (const uint4 *)src, ld / 16, (D * es + 15) / 16, top, place, (uint4 *)dst, ldo / 16);
}

__global__ void __launch_bounds__(256)
skn_gather_experts_kernel(float *x, int64_t ldx, int D, float alpha, int top, const int32_t *place, const float *weight, skn_rows_out y) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int64_t m = blockIdx.x;
    // (rows are padded to 8 columns: the padding of x takes the zeros of y's)
    for (int i = threadIdx.x * 4; i < D; i += 1024) {
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int k = 0; k < top; ++k) {
            const int64_t r = place[m * top + k];
            const float w = weight[m * top + k];
            float4 v;
            if (y.y32) v = *reinterpret_cast<const float4 *>(y.y32 + r * y.ld32 + i);
            else {
                const uint2 u = *reinterpret_cast<const uint2 *>(y.y16 + r * y.ld16 + i);
                v = make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xFFFF0000u));
            }
            a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
        }
        float4 *p = reinterpret_cast<float4 *>(x + m * ldx + i);
        float4 o = *p;
        o.x = fmaf(alpha, a.x, o.x); o.y = fmaf(alpha, a.y, o.y); o.z = fmaf(alpha, a.z, o.z); o.w = fmaf(alpha, a.w, o.w);
        *p = o;
    }
}

cudaError_t skn_launch_gather_experts(float *x, int64_t ldx, int M, int D, float alpha, int top, const int32_t *place, const float *weight,
                                      const skn_rows_out &y, cudaStream_t st) {
    return skn_launch_pdl(skn_gather_experts_kernel, dim3(M), dim3(256), 0, st, 1, x, ldx, D, alpha, top, place, weight, y);
}
