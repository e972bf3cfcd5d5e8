// Linear layers over dense bf16 weights [out][in] (row pitch a multiple of 16 bytes, rows zero-padded to it).
//
//  skn_dense_matvec_kernel   1 .. 4 activation rows, HBM-bound: x (fp32) is brought into shared memory once per CTA,
//                            with the RMS norm folded in; a warp streams two weight rows at a time.  The first
//                            weights of every warp are in flight before the kernel waits for its predecessor.
//  skn_dense_f32_kernel      any number of rows, fp32 products and sums on the CUDA cores (the 32-bit mode)
//  skn_dense_tc_kernel       tcgen05: a tile is 128 weight rows (TMEM lanes) x up to 256 tokens (TMEM columns), so
//                            the same kernel serves a batch of decode rows (narrow tiles, split-K over the SMs)
//                            and whole prompts (two accumulators: the epilogue of one tile runs under the
//                            products of the next)
#include "skn_dense.cuh"
#include "skn_tc.cuh"

__device__ __forceinline__ float dense_gelu_tanh(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <int EPI>
__device__ __forceinline__ void dense_store(const skn_epi &e, int64_t m, int64_t n, float v) {
    if (EPI == SKN_EPI_ADD) v += e.resid[m * e.ld_resid + n];
    if (EPI == SKN_EPI_RELU2) {
        v = fmaxf(v, 0.f);
        v *= v;
    }
    if (EPI == SKN_EPI_GELU_TABLE) {
        int64_t id = e.ids[m];
        if (id < 0 || id >= e.table_rows) id = 0;      // out-of-range ids read row 0, as the embedding does
        v = dense_gelu_tanh(v) * __bfloat162float(e.table[id * e.ld_table + e.table_col + n]);
    }
    if (e.y32) e.y32[m * e.ld_y32 + n] = v;
    if (e.y16) e.y16[m * e.ld_y16 + n] = __float2bfloat16_rn(v);
}

__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xFFFF0000u); }

// ---- matvec ------------------------------------------------------------------------------------------------
constexpr int MVD_THREADS = 512, MVD_WARPS = MVD_THREADS / 32, MVD_U = 4;

template <int MR, int EPI>
__global__ void __launch_bounds__(MVD_THREADS, 1)
skn_dense_matvec_kernel(const uint8_t *__restrict__ W, int64_t pitch, int N, int K, int m0, const float *__restrict__ x, int64_t ldx,
                        const float *__restrict__ xb, int64_t ldxb, int ka, const float *__restrict__ gain, float eps, skn_epi e) {
    extern __shared__ float xs[];                  // [MR][2 planes][K8 / 2]: quads 0 and 1 of every eight columns
    __shared__ float red[MVD_WARPS][MR];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int nv = (int)(pitch >> 4), K8 = nv * 8, half = K8 / 2;
    const int pairs = (N + 1) / 2;
    const int stride = gridDim.x * MVD_WARPS;
    int pair = warp * gridDim.x + blockIdx.x;

    uint4 wa[MVD_U], wb[MVD_U];
    auto load = [&](int p, int i0) {
        const bool two = 2 * p + 1 < N;
        const uint4 *ra = reinterpret_cast<const uint4 *>(W + (int64_t)(2 * p) * pitch);
        const uint4 *rb = reinterpret_cast<const uint4 *>(W + (int64_t)(2 * p + 1) * pitch);
#pragma unroll
        for (int u = 0; u < MVD_U; ++u) {
            const int i = i0 + u * 32 + lane;
            const bool in = i < nv;
            wa[u] = in ? __ldg(ra + i) : make_uint4(0u, 0u, 0u, 0u);
            wb[u] = in && two ? __ldg(rb + i) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    if (pair < pairs) load(pair, 0);
    skn_pdl_launch_dependents();
    skn_pdl_wait();

    float ss[MR];
#pragma unroll
    for (int m = 0; m < MR; ++m) {
        ss[m] = 0.f;
        const float *xr = x + (int64_t)(m0 + m) * ldx;
        const float *xbr = xb ? xb + (int64_t)(m0 + m) * ldxb - ka : xr;
        float *dst = xs + m * K8;
#pragma unroll 4
        for (int k = threadIdx.x; k < K8; k += MVD_THREADS) {
            float v = 0.f;
            if (k < K) v = __ldcg(k < ka ? xr + k : xbr + k);
            ss[m] = fmaf(v, v, ss[m]);
            if (gain && k < K) v *= __ldg(gain + k);
            dst[((k >> 2) & 1) * half + (k >> 3) * 4 + (k & 3)] = v;
        }
    }
    if (gain) {
#pragma unroll
        for (int m = 0; m < MR; ++m) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) ss[m] += __shfl_xor_sync(0xffffffffu, ss[m], o);
            if (lane == 0) red[warp][m] = ss[m];
        }
    }
    __syncthreads();
    float rs[MR];
#pragma unroll
    for (int m = 0; m < MR; ++m) {
        rs[m] = 1.f;
        if (gain) {
            float t = 0.f;
#pragma unroll
            for (int w = 0; w < MVD_WARPS; ++w) t += red[w][m];
            rs[m] = 1.f / sqrtf(t / (float)K + eps);
        }
    }

    float a0[MR], a1[MR];
#pragma unroll
    for (int m = 0; m < MR; ++m) a0[m] = a1[m] = 0.f;
    int i0 = 0;
    while (pair < pairs) {
#pragma unroll
        for (int u = 0; u < MVD_U; ++u) {
            const int i = i0 + u * 32 + lane;
            if (i < nv) {
                const uint4 p = wa[u], q = wb[u];
#pragma unroll
                for (int m = 0; m < MR; ++m) {
                    const float4 lo = *reinterpret_cast<const float4 *>(xs + m * K8 + i * 4);
                    const float4 hi = *reinterpret_cast<const float4 *>(xs + m * K8 + half + i * 4);
                    float s = a0[m], t = a1[m];
                    s = fmaf(bf_lo(p.x), lo.x, s); s = fmaf(bf_hi(p.x), lo.y, s); s = fmaf(bf_lo(p.y), lo.z, s); s = fmaf(bf_hi(p.y), lo.w, s);
                    s = fmaf(bf_lo(p.z), hi.x, s); s = fmaf(bf_hi(p.z), hi.y, s); s = fmaf(bf_lo(p.w), hi.z, s); s = fmaf(bf_hi(p.w), hi.w, s);
                    t = fmaf(bf_lo(q.x), lo.x, t); t = fmaf(bf_hi(q.x), lo.y, t); t = fmaf(bf_lo(q.y), lo.z, t); t = fmaf(bf_hi(q.y), lo.w, t);
                    t = fmaf(bf_lo(q.z), hi.x, t); t = fmaf(bf_hi(q.z), hi.y, t); t = fmaf(bf_lo(q.w), hi.z, t); t = fmaf(bf_hi(q.w), hi.w, t);
                    a0[m] = s;
                    a1[m] = t;
                }
            }
        }
        const int done = pair;
        i0 += 32 * MVD_U;
        const bool last = i0 >= nv;
        if (last) {
            i0 = 0;
            pair += stride;
        }
        if (pair < pairs) load(pair, i0);
        if (last) {
            float mine = 0.f;
#pragma unroll
            for (int m = 0; m < MR; ++m) {
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) {
                    a0[m] += __shfl_xor_sync(0xffffffffu, a0[m], o);
                    a1[m] += __shfl_xor_sync(0xffffffffu, a1[m], o);
                }
                if (lane == 2 * m) mine = a0[m] * rs[m];
                if (lane == 2 * m + 1) mine = a1[m] * rs[m];
                a0[m] = a1[m] = 0.f;
            }
            const int n = 2 * done + (lane & 1);
            if (lane < 2 * MR && n < N) dense_store<EPI>(e, m0 + (lane >> 1), n, mine);
        }
    }
}

template <int MR, int EPI>
static cudaError_t launch_mvd(skn_ctx *ctx, const skn_linear &l, int m0, cudaStream_t st) {
    auto kern = skn_dense_matvec_kernel<MR, EPI>;
    const int K8 = (int)(l.w->pitch / 2);
    const size_t smem = (size_t)MR * K8 * sizeof(float);
    static bool attr_done[64] = {false};
    if (!attr_done[ctx->device & 63]) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) return e;
        attr_done[ctx->device & 63] = true;
    }
    const int pairs = (int)((l.w->n_rows + 1) / 2);
    int grid = (pairs + MVD_WARPS - 1) / MVD_WARPS;
    // few rows: one warp per CTA has work, so that every SM takes part
    if (grid < ctx->sm_count) grid = pairs < ctx->sm_count ? pairs : ctx->sm_count;
    if (grid > ctx->sm_count) grid = ctx->sm_count;
    const int K = (int)l.w->n_cols;
    return skn_launch_pdl(kern, dim3(grid), dim3(MVD_THREADS), smem, st, 1, (const uint8_t *)l.w->d_blocks, l.w->pitch, (int)l.w->n_rows, K,
                          m0, l.x32, l.ld_x32, l.x32b, l.ld_x32b, l.x32b ? (int)l.k_a : K, l.gain, l.eps, l.epi);
}

template <int MR>
static cudaError_t dispatch_mvd(skn_ctx *ctx, const skn_linear &l, int m0, cudaStream_t st) {
    switch (l.epi.kind) {
    case SKN_EPI_STORE: return launch_mvd<MR, SKN_EPI_STORE>(ctx, l, m0, st);
    case SKN_EPI_ADD: return launch_mvd<MR, SKN_EPI_ADD>(ctx, l, m0, st);
    case SKN_EPI_RELU2: return launch_mvd<MR, SKN_EPI_RELU2>(ctx, l, m0, st);
    case SKN_EPI_GELU_TABLE: return launch_mvd<MR, SKN_EPI_GELU_TABLE>(ctx, l, m0, st);
    }
    return cudaErrorInvalidValue;
}

cudaError_t skn_launch_dense_matvec(skn_ctx *ctx, const skn_linear &l, cudaStream_t st) {
    const size_t row = (size_t)l.w->pitch * 2;            // one activation row in shared memory
    int fit = (int)((size_t)200 * 1024 / row);
    if (fit < 1) return cudaErrorNotSupported;
    for (int m0 = 0; m0 < l.M;) {
        const int left = l.M - m0;
        int mr = left >= 4 && fit >= 4 ? 4 : left >= 2 && fit >= 2 ? 2 : 1;
        const cudaError_t e = mr == 4 ? dispatch_mvd<4>(ctx, l, m0, st) : mr == 2 ? dispatch_mvd<2>(ctx, l, m0, st) : dispatch_mvd<1>(ctx, l, m0, st);
        if (e != cudaSuccess) return e;
        m0 += mr;
    }
    return cudaSuccess;
}

// ---- fp32 ----------------------------------------------------------------------------------------------------
// 64 tokens x 64 weight rows per CTA, K in steps of 16; a thread owns 4 x 4 outputs
constexpr int F32_BM = 64, F32_BN = 64, F32_BK = 16;

template <int EPI>
__global__ void __launch_bounds__(256)
skn_dense_f32_kernel(const uint8_t *__restrict__ W, int64_t pitch, int N, int K, int M, const float *__restrict__ x, int64_t ldx,
                     const float *__restrict__ xb, int64_t ldxb, int ka, skn_epi e) {
    __shared__ float xt[F32_BK][F32_BM + 4], wt[F32_BK][F32_BN + 4];
    const int m0 = blockIdx.y * F32_BM, n0 = blockIdx.x * F32_BN;
    const int tm = (threadIdx.x >> 4) * 4, tn = (threadIdx.x & 15) * 4;
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += F32_BK) {
#pragma unroll
        for (int i = threadIdx.x; i < F32_BM * F32_BK; i += 256) {
            const int r = i / F32_BK, c = i % F32_BK, k = k0 + c, m = m0 + r, n = n0 + r;
            float v = 0.f, w = 0.f;
            if (k < K) {
                if (m < M) v = __ldcg(k < ka ? x + (int64_t)m * ldx + k : xb + (int64_t)m * ldxb + k - ka);
                if (n < N) w = __bfloat162float(reinterpret_cast<const __nv_bfloat16 *>(W + (int64_t)n * pitch)[k]);
            }
            xt[c][r] = v;
            wt[c][r] = w;
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < F32_BK; ++c) {
            const float4 a = *reinterpret_cast<const float4 *>(&xt[c][tm]), b = *reinterpret_cast<const float4 *>(&wt[c][tn]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (m0 + tm + i < M && n0 + tn + j < N) dense_store<EPI>(e, m0 + tm + i, n0 + tn + j, acc[i][j]);
}

cudaError_t skn_launch_dense_f32(skn_ctx *, const skn_linear &l, cudaStream_t st) {
    const int N = (int)l.w->n_rows, K = (int)l.w->n_cols;
    const dim3 grid((N + F32_BN - 1) / F32_BN, (l.M + F32_BM - 1) / F32_BM);
    const int ka = l.x32b ? (int)l.k_a : K;
#define F32_CASE(EPI) \
    case EPI: \
        return skn_launch_pdl(skn_dense_f32_kernel<EPI>, grid, dim3(256), 0, st, 1, (const uint8_t *)l.w->d_blocks, l.w->pitch, N, K, l.M, \
                              l.x32, l.ld_x32, l.x32b, l.ld_x32b, ka, l.epi)
    switch (l.epi.kind) {
        F32_CASE(SKN_EPI_STORE);
        F32_CASE(SKN_EPI_ADD);
        F32_CASE(SKN_EPI_RELU2);
        F32_CASE(SKN_EPI_GELU_TABLE);
    }
#undef F32_CASE
    return cudaErrorInvalidValue;
}

// ---- tensor cores ------------------------------------------------------------------------------------------------
constexpr int DTC_BM = 128, DTC_BK = 64;
constexpr int DTC_A_BYTES = DTC_BM * DTC_BK * 2;
constexpr int DTC_THREADS = 6 * 32;              // four epilogue warps, one MMA warp, one TMA warp
constexpr int DTC_SMEM = 208 * 1024;
constexpr int DTC_MAX_STAGES = 8;

__device__ __forceinline__ void dtc_barrier_epilogue() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

template <int EPI>
__global__ void __launch_bounds__(DTC_THREADS, 1)
skn_dense_tc_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x, int N, int K, int M, int NT,
                    int stages, int splits, float *__restrict__ partial, unsigned *__restrict__ tickets, skn_epi e,
                    int32_t *__restrict__ status) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ uint64_t full_bar[DTC_MAX_STAGES], empty_bar[DTC_MAX_STAGES], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_slot, last_flag;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int stage_bytes = DTC_A_BYTES + NT * DTC_BK * 2;
    const int acc_cols = NT < 32 ? 32 : NT;
    uint32_t tmem_cols = 32;
    while ((int)tmem_cols < 2 * acc_cols) tmem_cols *= 2;
    const int ksteps = (K + DTC_BK - 1) / DTC_BK;
    const int mt = (M + NT - 1) / NT, nt = (N + DTC_BM - 1) / DTC_BM;
    const int units = mt * nt * splits;          // token tiles fastest, then splits, then weight tiles

    if (threadIdx.x == 0) {
        for (int s = 0; s < stages; ++s) {
            skn_mbar_init(&full_bar[s], 1);
            skn_mbar_init(&empty_bar[s], 1);
        }
        for (int b = 0; b < 2; ++b) {
            skn_mbar_init(&acc_full[b], 1);
            skn_mbar_init(&acc_empty[b], 4);
        }
        skn_fence_mbar_init();
    }
    if (warp == 4) tc_alloc(&tmem_slot, tmem_cols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    skn_pdl_launch_dependents();
    skn_pdl_wait();

    if (warp == 5) {
        if (lane == 0) {
            bool ok = true;
            int it = 0;
            for (int u = blockIdx.x; u < units && ok; u += gridDim.x) {
                const int m0 = (u % mt) * NT, sp = (u / mt) % splits, n0 = (u / mt / splits) * DTC_BM;
                const int kb = (int)((int64_t)ksteps * sp / splits), ke = (int)((int64_t)ksteps * (sp + 1) / splits);
                for (int k = kb; k < ke; ++k, ++it) {
                    const int s = it % stages;
                    if (!skn_mbar_wait(&empty_bar[s], ((uint32_t)(it / stages) & 1u) ^ 1u)) {
                        atomicExch(status, SKN_ERR_TIMEOUT);
                        ok = false;
                        break;
                    }
                    uint8_t *a = smem + (size_t)s * stage_bytes;
                    skn_mbar_expect_tx(&full_bar[s], (uint32_t)stage_bytes);
                    tc_tma_load_2d(a, &tmap_w, k * DTC_BK, n0, &full_bar[s]);
                    tc_tma_load_2d(a + DTC_A_BYTES, &tmap_x, k * DTC_BK, m0, &full_bar[s]);
                }
            }
            // the last copies have landed before this CTA ends: drain the stages still in flight
            for (int j = it > stages ? it - stages : 0; j < it && ok; ++j)
                if (!skn_mbar_wait(&full_bar[j % stages], (uint32_t)(j / stages) & 1u)) {
                    atomicExch(status, SKN_ERR_TIMEOUT);
                    ok = false;
                }
        }
    } else if (warp == 4) {
        if (lane == 0) {
            const uint32_t idesc = tc_idesc(DTC_BM, NT);
            bool ok = true;
            int it = 0, tile = 0;
            for (int u = blockIdx.x; u < units && ok; u += gridDim.x, ++tile) {
                const int sp = (u / mt) % splits;
                const int kb = (int)((int64_t)ksteps * sp / splits), ke = (int)((int64_t)ksteps * (sp + 1) / splits);
                const int b = tile & 1;
                if (!skn_mbar_wait(&acc_empty[b], ((uint32_t)(tile >> 1) & 1u) ^ 1u)) {
                    atomicExch(status, SKN_ERR_TIMEOUT);
                    break;
                }
                tc_fence_after();
                const uint32_t d = tmem + (uint32_t)(b * acc_cols);
                for (int k = kb; k < ke; ++k, ++it) {
                    const int s = it % stages;
                    if (!skn_mbar_wait(&full_bar[s], (uint32_t)(it / stages) & 1u)) {
                        atomicExch(status, SKN_ERR_TIMEOUT);
                        ok = false;
                        break;
                    }
                    tc_fence_after();
                    const uint32_t base = skn_smem_u32(smem + (size_t)s * stage_bytes);
                    const uint64_t ad = tc_smem_desc(base), bd = tc_smem_desc(base + DTC_A_BYTES);
#pragma unroll
                    for (int j = 0; j < DTC_BK / 16; ++j) tc_mma_bf16(d, ad + 2 * j, bd + 2 * j, idesc, (k > kb || j > 0) ? 1u : 0u);
                    tc_commit(&empty_bar[s]);
                }
                tc_commit(&acc_full[b]);
            }
        }
    } else {
        // epilogue: TMEM lane = weight row, column = token; a warp's store covers 32 consecutive outputs of one token
        bool ok = true;
        int tile = 0;
        for (int u = blockIdx.x; u < units; u += gridDim.x, ++tile) {
            const int m0 = (u % mt) * NT, sp = (u / mt) % splits, nti = u / mt / splits, n0 = nti * DTC_BM;
            const int b = tile & 1;
            if (ok && !skn_mbar_wait(&acc_full[b], (uint32_t)(tile >> 1) & 1u)) {
                if (lane == 0) atomicExch(status, SKN_ERR_TIMEOUT);
                ok = false;
            }
            tc_fence_after();
            const int n = n0 + warp * 32 + lane;
            const int cols = min(NT, M - m0);
            const uint32_t src = tmem + (uint32_t)(b * acc_cols) + ((uint32_t)(warp * 32) << 16);
            const int tidx = nti * mt + u % mt;
            float *pbase = partial + ((size_t)tidx * splits) * NT * DTC_BM + warp * 32 + lane;
#pragma unroll 1
            for (int c0 = 0; c0 < cols; c0 += 32) {
                uint32_t acc[32];
                tc_ld32(src + c0, acc);
                if (splits == 1) {
                    if (n < N && ok) {
                        if (cols - c0 >= 32) {
#pragma unroll
                            for (int c = 0; c < 32; ++c) dense_store<EPI>(e, m0 + c0 + c, n, __uint_as_float(acc[c]));
                        } else {
#pragma unroll
                            for (int c = 0; c < 32; ++c)
                                if (c0 + c < cols) dense_store<EPI>(e, m0 + c0 + c, n, __uint_as_float(acc[c]));
                        }
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < 32; ++c)
                        if (c0 + c < cols) __stcg(pbase + ((size_t)sp * NT + c0 + c) * DTC_BM, __uint_as_float(acc[c]));
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) skn_mbar_arrive(&acc_empty[b]);
            if (splits > 1) {
                // the split that arrives last at its tile adds the partial sums in split order
                __threadfence();
                dtc_barrier_epilogue();
                if (threadIdx.x == 0) last_flag = atomicAdd(&tickets[tidx], 1u) == (unsigned)(splits - 1);
                dtc_barrier_epilogue();
                if (last_flag) {
                    __threadfence();
                    for (int c = 0; c < cols; ++c) {
                        float v = 0.f;
                        for (int s = 0; s < splits; ++s) v += __ldcg(pbase + ((size_t)s * NT + c) * DTC_BM);
                        if (n < N && ok) dense_store<EPI>(e, m0 + c, n, v);
                    }
                    if (threadIdx.x == 0) tickets[tidx] = 0;
                }
                dtc_barrier_epilogue();
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 4) {
        __syncwarp();
        tc_fence_after();
        tc_dealloc(tmem, tmem_cols);
    }
}

template <int EPI>
static cudaError_t launch_dtc(skn_ctx *ctx, const skn_linear &l, const skn_dense_ws &ws, cudaStream_t st) {
    auto kern = skn_dense_tc_kernel<EPI>;
    static bool attr_done[64] = {false};
    if (!attr_done[ctx->device & 63]) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, DTC_SMEM + 1024);
        if (e != cudaSuccess) return e;
        attr_done[ctx->device & 63] = true;
    }
    const int N = (int)l.w->n_rows, K = (int)l.w->n_cols, M = l.M, sms = ctx->sm_count;
    const int nt = (N + DTC_BM - 1) / DTC_BM;
    // token tile: the narrowest that covers M, at most 256; halved while that leaves SMs without a tile
    int NT = 16;
    while (NT < 256 && NT < M) NT *= 2;
    while (NT > 64 && nt * ((M + NT - 1) / NT) < sms) NT /= 2;
    const int mt = (M + NT - 1) / NT, ksteps = (K + DTC_BK - 1) / DTC_BK;
    int splits = 1;
    if (mt * nt < sms && mt * nt <= SKN_DENSE_MAX_TILES) {
        splits = sms / (mt * nt);
        if (splits > ksteps / 4) splits = ksteps / 4;                // at least four K steps each
        if (splits > 16) splits = 16;
        while (splits > 1 && (size_t)mt * nt * splits * NT * DTC_BM > SKN_DENSE_WS_FLOATS) --splits;
        if (splits < 1) splits = 1;
    }
    const int stage_bytes = DTC_A_BYTES + NT * DTC_BK * 2;
    int stages = DTC_SMEM / stage_bytes;
    if (stages > DTC_MAX_STAGES) stages = DTC_MAX_STAGES;
    CUtensorMap tw, tx;
    cudaError_t e = skn_tmap_bf16(l.w->d_blocks, N, K, l.w->pitch, DTC_BM, &tw);
    if (e == cudaSuccess) e = skn_tmap_bf16(l.x16, M, K, l.ld_x16 * 2, NT, &tx);
    if (e != cudaSuccess) return e;
    const int units = mt * nt * splits;
    return skn_launch_pdl(kern, dim3(units < sms ? units : sms), dim3(DTC_THREADS), (size_t)stages * stage_bytes + 1024, st, 1, tw, tx, N, K, M, NT,
                          stages, splits, ws.partial, ws.tickets, l.epi, ctx->d_status);
}

cudaError_t skn_launch_dense_tc(skn_ctx *ctx, const skn_linear &l, const skn_dense_ws &ws, cudaStream_t st) {
    if (l.ld_x16 % 8) return cudaErrorInvalidValue;
    switch (l.epi.kind) {
    case SKN_EPI_STORE: return launch_dtc<SKN_EPI_STORE>(ctx, l, ws, st);
    case SKN_EPI_ADD: return launch_dtc<SKN_EPI_ADD>(ctx, l, ws, st);
    case SKN_EPI_RELU2: return launch_dtc<SKN_EPI_RELU2>(ctx, l, ws, st);
    case SKN_EPI_GELU_TABLE: return launch_dtc<SKN_EPI_GELU_TABLE>(ctx, l, ws, st);
    }
    return cudaErrorInvalidValue;
}
