// Linear layers over dense bf16 weights [out][in] (row pitch a multiple of 16 bytes, rows zero-padded to it).
//
//  skn_dense_matvec_kernel   1 .. 4 activation rows (fp32), HBM-bound: weight rows stream through shared memory in bulk
//                            copies, the RMS norm of x is folded in
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
// 0.5 (1 + tanh u) = 1 / (1 + exp(-2 u)); relative error a few 1e-7
__device__ __forceinline__ float dense_gelu_exp(float z) {
    return __fdividef(z, 1.f + __expf(fminf(-1.5957691216057308f * (z + 0.044715f * z * z * z), 80.f)));
}
__device__ __forceinline__ float dense_silu(float z) { return __fdividef(z, 1.f + __expf(fminf(-z, 80.f))); }

template <int EPI>
__device__ __forceinline__ void dense_store(const skn_epi &e, int64_t m, int64_t n, float v) {
    if (EPI == SKN_EPI_ADD) v = fmaf(e.alpha, v, e.resid[m * e.ld_resid + n]);
    if (EPI == SKN_EPI_GELU_TAIL && n >= e.n_act) {
        v = dense_gelu_exp(v);
        if (e.act32) e.act32[m * e.ld_act32 + n - e.n_act] = v;
        if (e.act16) e.act16[m * e.ld_act16 + n - e.n_act] = __float2bfloat16_rn(v);
        return;
    }
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

__device__ __forceinline__ void dense_put(const skn_epi &e, int64_t m, int64_t n, float v) {
    if (e.y32) e.y32[m * e.ld_y32 + n] = v;
    if (e.y16) e.y16[m * e.ld_y16 + n] = __float2bfloat16_rn(v);
}
// gate and up of an activation column
__device__ __forceinline__ void dense_put_silu(const skn_epi &e, int64_t m, int64_t n, float gate, float up) {
    float v = dense_silu(gate) * up;
    if (e.act_scale) v *= e.act_scale[(n - e.n_act) / e.scale_rows];
    const int64_t c = (n - e.n_act) >> 1;
    if (e.act32) e.act32[m * e.ld_act32 + c] = v;
    if (e.act16) e.act16[m * e.ld_act16 + c] = __float2bfloat16_rn(v);
}
// angle of the pair that row n belongs to; false: it passes unchanged
__device__ __forceinline__ bool dense_angle(const skn_epi &e, int64_t m, int64_t n, float2 &cs) {
    const int i = ((int)(n % e.rot_head) - e.rot_lo) >> 1;
    if (i < 0 || i >= e.rot.half) return false;
    cs = __ldcg(e.rot.table + m * e.rot.ld + i);
    return true;
}
// weight rows n (even) and n + 1 of token m, for the epilogues that work on pairs
template <int EPI>
__device__ __forceinline__ void dense_store_pair(const skn_epi &e, int64_t m, int64_t n, float a, float b, bool both) {
    if (EPI == SKN_EPI_SILU_TAIL && n >= e.n_act) {
        if (both) dense_put_silu(e, m, n, a, b);
        return;
    }
    float2 cs;
    if (EPI == SKN_EPI_ROTATE && both && dense_angle(e, m, n, cs)) {
        const float u = a;
        a = u * cs.x - b * cs.y;
        b = b * cs.x + u * cs.y;
    }
    dense_put(e, m, n, a);
    if (both) dense_put(e, m, n + 1, b);
}

// NC consecutive tokens m .. of weight row n: everything the epilogue reads is loaded before the first store
template <int EPI, int NC>
__device__ __forceinline__ void dense_store_run(const skn_epi &e, int64_t m, int64_t n, float (&v)[NC], int count) {
    if (EPI == SKN_EPI_ADD) {
        float r[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) r[c] = c < count ? e.resid[(m + c) * e.ld_resid + n] : 0.f;
#pragma unroll
        for (int c = 0; c < NC; ++c) v[c] = fmaf(e.alpha, v[c], r[c]);
    }
    if (EPI == SKN_EPI_GELU_TAIL && n >= e.n_act) {
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            if (c >= count) continue;
            const float g = dense_gelu_exp(v[c]);
            if (e.act32) e.act32[(m + c) * e.ld_act32 + n - e.n_act] = g;
            if (e.act16) e.act16[(m + c) * e.ld_act16 + n - e.n_act] = __float2bfloat16_rn(g);
        }
        return;
    }
    if (EPI == SKN_EPI_GELU_TABLE) {
        float r[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            int64_t id = c < count ? e.ids[m + c] : 0;
            if (id < 0 || id >= e.table_rows) id = 0;
            r[c] = __bfloat162float(e.table[id * e.ld_table + e.table_col + n]);
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) v[c] = dense_gelu_tanh(v[c]) * r[c];
    }
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        if (EPI == SKN_EPI_RELU2) {
            v[c] = fmaxf(v[c], 0.f);
            v[c] *= v[c];
        }
        if (c < count) {
            if (e.y32) e.y32[(m + c) * e.ld_y32 + n] = v[c];
            if (e.y16) e.y16[(m + c) * e.ld_y16 + n] = __float2bfloat16_rn(v[c]);
        }
    }
}

// NC tokens of bf16 rows, the whole warp together (lane l: row n = (even base) + l): neighbouring lanes trade every other token, so that a
// lane stores two columns at once.  y: column n of token m; `in` marks the rows that exist, in pairs.
template <int NC>
__device__ __forceinline__ void dense_put_packed(__nv_bfloat16 *y, int64_t ld, int64_t n, const float (&v)[NC], int count, bool in) {
    const bool odd = n & 1;
    uint32_t *p = reinterpret_cast<uint32_t *>(y - (odd ? 1 : 0)) + (odd ? ld / 2 : 0);
#pragma unroll
    for (int c = 0; c < NC; c += 2) {
        const float got = __shfl_xor_sync(0xffffffffu, odd ? v[c] : v[c + 1], 1);
        const uint32_t w = odd ? tc_pack_bf16(got, v[c + 1]) : tc_pack_bf16(v[c], got);
        if (in && c + (odd ? 1 : 0) < count) *p = w;
        p += ld;                                   // two tokens of ld / 2 words
    }
}
__device__ __forceinline__ bool dense_packs(const __nv_bfloat16 *y16, int64_t ld, const float *y32, int N) {
    return N % 4 == 0 && y16 && !y32 && ld % 2 == 0 && (reinterpret_cast<uintptr_t>(y16) & 3) == 0;
}

// NC tokens of rows (gate, up), a warp of activation rows only (n - n_act of its first lane is a multiple of 4).  The lanes of a pair take a
// token each, then lanes two apart trade tokens, so that a lane stores two columns of every fourth token.
template <int NC>
__device__ __forceinline__ void dense_put_silu_packed(const skn_epi &e, int64_t m, int64_t n, const float (&v)[NC], int count, bool in) {
    const bool odd = n & 1, high = (n >> 1) & 1;
    const int t0 = (odd ? 1 : 0) + (high ? 2 : 0);
    uint32_t *p = reinterpret_cast<uint32_t *>(e.act16 + (m + t0) * e.ld_act16 + (((n & ~(int64_t)3) - e.n_act) >> 1));
#pragma unroll
    for (int c = 0; c < NC; c += 4) {
        float f[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const float a = v[c + 2 * x], b = v[c + 2 * x + 1], got = __shfl_xor_sync(0xffffffffu, odd ? a : b, 1);
            f[x] = odd ? dense_silu(got) * b : dense_silu(a) * got;
        }
        const float got = __shfl_xor_sync(0xffffffffu, high ? f[0] : f[1], 2);
        const uint32_t w = high ? tc_pack_bf16(got, f[1]) : tc_pack_bf16(f[0], got);
        if (in && c + t0 < count) *p = w;
        p += e.ld_act16 * 2;                       // four tokens of ld / 2 words
    }
}

// The pair epilogues in general, the whole warp together: lane l holds row n = (even base) + l, `in` marks the rows that exist.
template <int EPI, int NC>
__device__ __forceinline__ void dense_store_run_pairs(const skn_epi &e, int N, int64_t m, int64_t n, float (&v)[NC], int count, bool in) {
    const bool odd = n & 1;
    if (EPI == SKN_EPI_ROTATE) {
        // the angles of the run are loaded before its first store
        const int i = ((int)(n % e.rot_head) - e.rot_lo) >> 1;
        const bool turn = in && i >= 0 && i < e.rot.half;
        float2 cs[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) cs[c] = turn && c < count ? __ldcg(e.rot.table + (m + c) * e.rot.ld + i) : make_float2(1.f, 0.f);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const float other = __shfl_xor_sync(0xffffffffu, v[c], 1);
            v[c] = odd ? v[c] * cs[c].x + other * cs[c].y : v[c] * cs[c].x - other * cs[c].y;
        }
        if (dense_packs(e.y16, e.ld_y16, e.y32, N)) {
            dense_put_packed(e.y16 + m * e.ld_y16 + n, e.ld_y16, n, v, count, in);
            return;
        }
#pragma unroll
        for (int c = 0; c < NC; ++c)
            if (c < count && in) dense_put(e, m + c, n, v[c]);
        return;
    }
    const bool act = n >= e.n_act;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        const float other = __shfl_xor_sync(0xffffffffu, v[c], 1);
        if (c >= count || !in) continue;
        if (!act) dense_put(e, m + c, n, v[c]);
        else if (!odd) dense_put_silu(e, m + c, n, v[c], other);
    }
}

// A run of NC tokens of the warp's 32 rows (lane l: row n, of N), in the quickest form that its destination allows
template <int EPI, int NC>
__device__ __forceinline__ void dense_store_warp(const skn_epi &e, int N, int64_t m, int64_t n, float (&v)[NC], int count, bool ok) {
    const bool in = n < N && ok;
    const int64_t first = n - (threadIdx.x & 31);
    if constexpr (EPI == SKN_EPI_STORE || EPI == SKN_EPI_RELU2) {
        if (dense_packs(e.y16, e.ld_y16, e.y32, N)) {
            if (EPI == SKN_EPI_RELU2)
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    v[c] = fmaxf(v[c], 0.f);
                    v[c] *= v[c];
                }
            dense_put_packed(e.y16 + m * e.ld_y16 + n, e.ld_y16, n, v, count, in);
            return;
        }
    }
    if constexpr (EPI == SKN_EPI_GELU_TAIL) {
        if (first >= e.n_act && e.n_act % 2 == 0 && dense_packs(e.act16, e.ld_act16, e.act32, N)) {
#pragma unroll
            for (int c = 0; c < NC; ++c) v[c] = dense_gelu_exp(v[c]);
            dense_put_packed(e.act16 + m * e.ld_act16 + n - e.n_act, e.ld_act16, n, v, count, in);
            return;
        }
    }
    if constexpr (EPI == SKN_EPI_SILU_TAIL) {
        if (first >= e.n_act && e.n_act % 4 == 0 && !e.act_scale && dense_packs(e.act16, e.ld_act16, e.act32, N)) {
            dense_put_silu_packed(e, m, n, v, count, in);
            return;
        }
        if (first + 31 < e.n_act) {                // none of the rows is activated
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (c < count && in) dense_put(e, m + c, n, v[c]);
            return;
        }
    }
    if constexpr (skn_epi_pairs(EPI)) dense_store_run_pairs<EPI, NC>(e, N, m, n, v, count, in);
    else if (in) dense_store_run<EPI, NC>(e, m, n, v, count);
}

// experts as groups of rows: first tile of each in tiles of NT rows (start[E]: their number), by one warp
__device__ __forceinline__ void dense_group_tiles(const int32_t *offset, int E, int NT, int *start, int *off) {
    const int lane = threadIdx.x & 31;
    int base = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
        const int e = e0 + lane;
        const int lo = e < E ? __ldcg(offset + e) : 0, hi = e < E ? __ldcg(offset + e + 1) : 0;
        int t = (hi - lo + NT - 1) / NT;
        const int own = t;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int y = __shfl_up_sync(0xffffffffu, t, o);
            if (lane >= o) t += y;
        }
        if (e < E) {
            start[e] = base + t - own;
            off[e] = lo;
            if (e == E - 1) off[E] = hi;
        }
        base += __shfl_sync(0xffffffffu, t, 31);
    }
    if (lane == 0) start[E] = base;
}
// expert of tile t
__device__ __forceinline__ int dense_group_of(const int *start, int E, int t) {
    int lo = 0, hi = E - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (start[mid] <= t) lo = mid;
        else hi = mid - 1;
    }
    return lo;
}

__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xFFFF0000u); }

// ---- matvec ------------------------------------------------------------------------------------------------
// CTA b owns the weight rows [b N / grid, (b + 1) N / grid): a producer warp streams them, a few rows per bulk copy, through
// a ring of shared-memory stages and starts before the kernel waits for its predecessor; eight warps each take an eighth of
// the columns of every row.  Their partial sums meet in shared memory, 128 rows at a time.  One activation row lives in
// registers (UU vectors of eight columns per lane), more rows in shared memory (UU = 0).
// EXT: a norm of a part of the columns, or rows longer than the registers hold, taken in column pieces: one piece after the other
// for all rows of the CTA (at most MVD_ROWS), the partial sums waiting in shared memory.
// PICK: the weight rows, or pieces of them, belong to experts that a kernel before chose, so the stream of those starts after
// the dependency wait.
constexpr int MVD_WARPS = 8, MVD_THREADS = (MVD_WARPS + 1) * 32, MVD_ROWS = 128;
constexpr int MVD_RING = 96 * 1024, MVD_MAX_STAGES = 24;
// dynamic shared memory beside the partial sums of MR rows
constexpr int mvd_smem(int mr) { return 224 * 1024 - mr * 2 * MVD_WARPS * MVD_ROWS * 4; }
// rows of a stage: about 16 KB of weights
__host__ __device__ constexpr int mvd_stage_rows(int mr, int uu) { return uu == 0 ? (mr > 1 ? 2 : 1) : uu == 1 ? 4 : uu == 2 ? 2 : 1; }

__device__ __forceinline__ void mvd_barrier() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

__device__ __forceinline__ void dense_store_any(const skn_epi &e, int64_t m, int64_t n, float v) {
    switch (e.kind) {
    case SKN_EPI_ADD: dense_store<SKN_EPI_ADD>(e, m, n, v); break;
    case SKN_EPI_RELU2: dense_store<SKN_EPI_RELU2>(e, m, n, v); break;
    case SKN_EPI_GELU_TABLE: dense_store<SKN_EPI_GELU_TABLE>(e, m, n, v); break;
    case SKN_EPI_GELU_TAIL: dense_store<SKN_EPI_GELU_TAIL>(e, m, n, v); break;
    default: dense_store<SKN_EPI_STORE>(e, m, n, v); break;
    }
}

__device__ __forceinline__ float mvd_dot8(const uint4 &w, const float4 &lo, const float4 &hi, float a) {
    a = fmaf(bf_lo(w.x), lo.x, a); a = fmaf(bf_hi(w.x), lo.y, a); a = fmaf(bf_lo(w.y), lo.z, a); a = fmaf(bf_hi(w.y), lo.w, a);
    a = fmaf(bf_lo(w.z), hi.x, a); a = fmaf(bf_hi(w.z), hi.y, a); a = fmaf(bf_lo(w.w), hi.z, a); return fmaf(bf_hi(w.w), hi.w, a);
}
// row of the eight whose sum this lane holds after the joint reduction
__device__ __forceinline__ int mvd_row(int lane) { return ((lane >> 4) & 1) * 4 + ((lane >> 3) & 1) * 2 + ((lane >> 2) & 1); }

struct mvd_pick {
    const int32_t *expert;
    const uint8_t *w2;                  // SKN_PICK_COLS
    int64_t pitch1, pitch2;             // SKN_PICK_COLS: bytes that w and each expert have in a joint row
    int n, rows_per;
};
struct mvd_norm {
    const float *gain;
    float eps;
    int cols, parts;                    // cols 0: the whole row
};

template <int MR, int UU, int PICK, bool PAIRS, bool EXT>
__global__ void __launch_bounds__(MVD_THREADS, 2)
skn_dense_matvec_kernel(const uint8_t *__restrict__ W, int64_t wld, int64_t row_bytes, int n_pieces, int64_t pitch, int N, int K, int m0, const float *x,
                        int64_t ldx, const float *xb, int64_t ldxb, int ka, mvd_norm nm, mvd_pick pk, int stages, skn_epi e, int32_t *status) {
    extern __shared__ __align__(128) uint8_t ring[];
    constexpr int GR = mvd_stage_rows(MR, UU);
    __shared__ uint64_t full_bar[MVD_MAX_STAGES], empty_bar[MVD_MAX_STAGES];
    __shared__ float red[MVD_WARPS][MR], part[2][MR][MVD_WARPS][MVD_ROWS], psum[EXT ? MR : 1][MVD_WARPS][EXT ? SKN_NORM_PARTS : 1];
    const float *__restrict__ gain = nm.gain;
    const bool partial = EXT && gain && nm.cols > 0;
    const int pieces = EXT ? n_pieces : 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int nv = (int)(pitch >> 4), K8 = nv * 8, half = K8 / 2;           // vectors of a piece (of the row, when there is one)
    const int q_rows = PAIRS ? 2 : 1, nq = (N + q_rows - 1) / q_rows;     // pairs of rows stay together
    const int r0 = min(N, q_rows * (int)((int64_t)nq * blockIdx.x / gridDim.x)), r1 = min(N, q_rows * (int)((int64_t)nq * (blockIdx.x + 1) / gridDim.x));
    const int steps = (r1 - r0 + GR - 1) / GR;
    const size_t stage_bytes = (size_t)GR * pitch;
    if (threadIdx.x == 0) {
        for (int s = 0; s < stages; ++s) {
            skn_mbar_init(&full_bar[s], 1);
            skn_mbar_init(&empty_bar[s], MVD_WARPS);
        }
        skn_fence_mbar_init();
    }
    __syncthreads();
    if (warp == MVD_WARPS) {
        if constexpr (PICK == SKN_PICK_NONE && !EXT) {
            if (lane == 0) {
                int s = 0;
                uint32_t phase = 1;
                for (int i = 0; i < steps; ++i) {
                    const int row = r0 + i * GR;
                    if (!skn_mbar_wait(&empty_bar[s], phase)) {
                        atomicExch(status, SKN_ERR_TIMEOUT);
                        break;
                    }
                    const uint32_t bytes = (uint32_t)(min(GR, r1 - row) * pitch);
                    skn_mbar_expect_tx(&full_bar[s], bytes);
                    skn_bulk_g2s(ring + s * stage_bytes, W + (int64_t)row * pitch, bytes, &full_bar[s]);
                    if (++s == stages) {
                        s = 0;
                        phase ^= 1u;
                    }
                }
            }
            skn_pdl_wait();
            return;
        }
        // lane 0 keeps the ring; the copies of a stage are issued by as many lanes as there are pieces of rows in it
        int s = 0, early = 0;
        uint32_t phase = 1;
        const int64_t own = PICK == SKN_PICK_COLS ? pk.pitch1 : row_bytes;
        if constexpr (PICK == SKN_PICK_COLS) {
            // w's part of the first stages depends on no kernel before this one
            const int64_t first = min(pitch, row_bytes), n_own = min(first, own);
            for (; early < stages && early < steps; ++early) {
                const int row = r0 + early * GR, n = min(GR, r1 - row);
                if (lane == 0) skn_mbar_expect_tx(&full_bar[early], (uint32_t)(n * first));
                __syncwarp();
                if (lane < n) skn_bulk_g2s(ring + early * stage_bytes + lane * pitch, W + (row + lane) * wld, (uint32_t)n_own, &full_bar[early]);
            }
        }
        if constexpr (PICK != SKN_PICK_NONE) skn_pdl_wait();
        for (int i = 0, pc = 0; pc < pieces; ++pc) {
            const int64_t lo = pc * pitch, hi = min(row_bytes, lo + pitch);
            for (int g = 0; g < steps; ++g, ++i) {
                const int row = r0 + g * GR, n = min(GR, r1 - row);
                int good = 1;
                if (lane == 0 && i >= early) {
                    good = skn_mbar_wait(&empty_bar[s], phase);
                    if (good) skn_mbar_expect_tx(&full_bar[s], (uint32_t)(n * (hi - lo)));
                    else atomicExch(status, SKN_ERR_TIMEOUT);
                }
                if (!__shfl_sync(0xffffffffu, good, 0)) {
                    pc = pieces;
                    break;
                }
                uint8_t *dst = ring + s * stage_bytes;
                if constexpr (PICK == SKN_PICK_NONE) {
                    if (wld == hi - lo) {
                        if (lane == 0) skn_bulk_g2s(dst, W + row * wld, (uint32_t)(n * wld), &full_bar[s]);
                    } else if (lane < n) {
                        skn_bulk_g2s(dst + lane * pitch, W + (row + lane) * wld + lo, (uint32_t)(hi - lo), &full_bar[s]);
                    }
                } else if constexpr (PICK == SKN_PICK_ROWS) {
                    if (lane < n) {
                        const int r = row + lane, x = r / pk.rows_per;
                        skn_bulk_g2s(dst + lane * pitch, W + ((int64_t)__ldcg(pk.expert + x) * pk.rows_per + r - x * pk.rows_per) * wld, (uint32_t)pitch, &full_bar[s]);
                    }
                } else {
                    // segment 0 of a joint row is w's, segment x + 1 belongs to the picked expert x
                    for (int u = lane; u < n * (pk.n + 1); u += 32) {
                        const int jr = u / (pk.n + 1), x = u % (pk.n + 1) - 1;
                        const int64_t s0 = x < 0 ? 0 : own + x * pk.pitch2, s1 = x < 0 ? own : s0 + pk.pitch2, a = max(lo, s0), b = min(hi, s1);
                        if (a >= b || (x < 0 && i < early)) continue;
                        const uint8_t *src = x < 0 ? W + (row + jr) * wld : pk.w2 + ((int64_t)__ldcg(pk.expert + x) * N + row + jr) * pk.pitch2;
                        skn_bulk_g2s(dst + jr * pitch + (a - lo), src + (a - s0), (uint32_t)(b - a), &full_bar[s]);
                    }
                }
                if (++s == stages) {
                    s = 0;
                    phase ^= 1u;
                }
            }
        }
        skn_pdl_wait();
        return;
    }
    skn_pdl_wait();

    bool ok = true;
    int buf = 0, filled = 0, base = r0;            // rows base .. base + filled - 1 have partial sums in part[buf]
    int s = 0;
    uint32_t phase = 0;
    const uint4 *w = reinterpret_cast<const uint4 *>(ring);
    for (int pc = 0; pc < pieces; ++pc) {
        // this warp's columns: vectors v0 + lane + 32 u below v1 of the piece, which starts at vector vb of the row
        const int vb = pc * nv, nvp = min(nv, (int)(row_bytes >> 4) - vb), per = (nvp + MVD_WARPS - 1) / MVD_WARPS, v0 = warp * per, v1 = min(nvp, v0 + per);
        float4 xr[UU > 0 ? 2 * UU : 1];
        float *xs = reinterpret_cast<float *>(ring + stages * stage_bytes);     // UU = 0: [MR][2 planes][K8 / 2]: quads 0 and 1 of every eight columns
        float ss[MR];
        auto fetch = [&](int m, int k) {
            float v = 0.f;
            if (k < K) v = __ldcg(k < ka ? x + (int64_t)(m0 + m) * ldx + k : xb + (int64_t)(m0 + m) * ldxb + k - ka);
            return v;
        };
        if constexpr (UU > 0) {
            // rows that are whole aligned vectors (the usual case) are read 16 bytes at a time
            const bool vec = K % 8 == 0 && ka % 8 == 0 && ldx % 4 == 0 && ldxb % 4 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(xb)) & 15) == 0;
            float q = 0.f, vsq[UU];
#pragma unroll
            for (int u = 0; u < UU; ++u) {
                const int i = v0 + u * 32 + lane;
                vsq[u] = 0.f;
                float f[8];
                const int k = (vb + i) * 8;
                if (vec && i < v1) {
                    const float *p = k < ka ? x + (int64_t)m0 * ldx + k : xb + (int64_t)m0 * ldxb + k - ka;
                    *reinterpret_cast<float4 *>(f) = __ldcg(reinterpret_cast<const float4 *>(p));
                    *reinterpret_cast<float4 *>(f + 4) = __ldcg(reinterpret_cast<const float4 *>(p + 4));
                } else {
#pragma unroll
                    for (int j = 0; j < 8; ++j) f[j] = i < v1 ? fetch(0, k + j) : 0.f;
                }
#pragma unroll
                for (int j = 0; j < 8; ++j) vsq[u] = fmaf(f[j], f[j], vsq[u]);
                q += vsq[u];
                if (gain && i < v1 && (!partial || k < nm.cols)) {
                    if (vec) {
                        const float4 g0 = __ldg(reinterpret_cast<const float4 *>(gain + k)), g1 = __ldg(reinterpret_cast<const float4 *>(gain + k + 4));
                        f[0] *= g0.x; f[1] *= g0.y; f[2] *= g0.z; f[3] *= g0.w;
                        f[4] *= g1.x; f[5] *= g1.y; f[6] *= g1.z; f[7] *= g1.w;
                    } else {
#pragma unroll
                        for (int j = 0; j < 8; ++j)
                            if (k + j < K) f[j] *= __ldg(gain + k + j);
                    }
                }
                xr[2 * u] = make_float4(f[0], f[1], f[2], f[3]);
                xr[2 * u + 1] = make_float4(f[4], f[5], f[6], f[7]);
            }
            ss[0] = q;
            if (EXT && partial && pc == 0) {
                const int pv = nm.cols / nm.parts / 8;                     // vectors of a part
                for (int p = 0; p < nm.parts; ++p) {
                    float t = 0.f;
#pragma unroll
                    for (int u = 0; u < UU; ++u) {
                        const int i = v0 + u * 32 + lane;
                        if (i < v1 && i / pv == p) t += vsq[u];
                    }
#pragma unroll
                    for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
                    if (lane == 0) psum[0][warp][p] = t;
                }
            }
        } else {
#pragma unroll
            for (int m = 0; m < MR; ++m) {
                ss[m] = 0.f;
                for (int k = threadIdx.x; k < K8; k += MVD_WARPS * 32) {
                    float v = fetch(m, k);
                    ss[m] = fmaf(v, v, ss[m]);
                    if (gain && k < K && !partial) v *= __ldg(gain + k);
                    xs[m * K8 + ((k >> 2) & 1) * half + (k >> 3) * 4 + (k & 3)] = v;
                }
            }
            if (EXT && partial) {
                const int part_cols = nm.cols / nm.parts;
                mvd_barrier();
#pragma unroll
                for (int m = 0; m < MR; ++m)
                    for (int p = 0; p < nm.parts; ++p) {
                        float t = 0.f;
                        for (int k = p * part_cols + threadIdx.x; k < (p + 1) * part_cols; k += MVD_WARPS * 32) {
                            const float v = xs[m * K8 + ((k >> 2) & 1) * half + (k >> 3) * 4 + (k & 3)];
                            t = fmaf(v, v, t);
                        }
#pragma unroll
                        for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
                        if (lane == 0) psum[m][warp][p] = t;
                    }
            }
        }
#pragma unroll
        for (int m = 0; m < MR; ++m) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) ss[m] += __shfl_xor_sync(0xffffffffu, ss[m], o);
            if (lane == 0) red[warp][m] = ss[m];
        }
        mvd_barrier();
        float rs[MR];
#pragma unroll
        for (int m = 0; m < MR; ++m) {
            rs[m] = 1.f;
            if (gain && !partial) {
                float t = 0.f;
#pragma unroll
                for (int w = 0; w < MVD_WARPS; ++w) t += red[w][m];
                rs[m] = 1.f / sqrtf(t / (float)K + nm.eps);
            }
        }
        if (EXT && partial && pc == 0) {                // (the parts lie in the first piece)
            const int part_cols = nm.cols / nm.parts;
            auto scale = [&](int m, int p) {
                float t = 0.f;
#pragma unroll
                for (int w = 0; w < MVD_WARPS; ++w) t += psum[m][w][p];
                return 1.f / sqrtf(t / (float)part_cols + nm.eps);
            };
            if constexpr (UU > 0) {
#pragma unroll
                for (int u = 0; u < UU; ++u) {
                    const int k = (v0 + u * 32 + lane) * 8;
                    if (k < nm.cols) {
                        const float f = scale(0, k / part_cols);
                        xr[2 * u].x *= f; xr[2 * u].y *= f; xr[2 * u].z *= f; xr[2 * u].w *= f;
                        xr[2 * u + 1].x *= f; xr[2 * u + 1].y *= f; xr[2 * u + 1].z *= f; xr[2 * u + 1].w *= f;
                    }
                }
            } else {
#pragma unroll
                for (int m = 0; m < MR; ++m)
                    for (int p = 0; p < nm.parts; ++p) {
                        const float f = scale(m, p);
                        for (int k = p * part_cols + threadIdx.x; k < (p + 1) * part_cols; k += MVD_WARPS * 32)
                            xs[m * K8 + ((k >> 2) & 1) * half + (k >> 3) * 4 + (k & 3)] *= f * __ldg(gain + k);
                    }
                mvd_barrier();
            }
        }

        // eight rows at a time: their sums are reduced across the warp together (9 shuffles for 8 rows)
        const bool last = pc + 1 == pieces;
        filled = 0;
        for (int g0 = 0; g0 < r1 - r0; g0 += 8) {
            float acc[MR][8];
#pragma unroll
            for (int m = 0; m < MR; ++m)
#pragma unroll
                for (int j = 0; j < 8; ++j) acc[m][j] = 0.f;
            const int rows = min(8, r1 - r0 - g0);
            // the next launch comes in under the last rows: earlier, its own stream of weights delays this one's
            if (last && g0 + 16 >= r1 - r0 && g0 + 8 < r1 - r0) skn_pdl_launch_dependents();
#pragma unroll
            for (int j0 = 0; j0 < 8; j0 += GR) {
                if (j0 < rows) {
                    if (ok && !skn_mbar_wait(&full_bar[s], phase)) {
                        if (lane == 0) atomicExch(status, SKN_ERR_TIMEOUT);
                        ok = false;
                    }
                    // (rows past the CTA's last one are old bytes of the ring: multiplied, never stored)
                    if constexpr (UU > 0) {
                        float odd[GR] = {};            // two chains
#pragma unroll
                        for (int u = 0; u < UU; ++u) {
                            const int c = v0 + u * 32 + lane;
                            if (c < v1) {
#pragma unroll
                                for (int j = 0; j < GR; ++j) {
                                    float &t = (u & 1) ? odd[j] : acc[0][j0 + j];
                                    t = mvd_dot8(w[j * nv + c], xr[2 * u], xr[2 * u + 1], t);
                                }
                            }
                        }
#pragma unroll
                        for (int j = 0; j < GR; ++j) acc[0][j0 + j] += odd[j];
                    } else {
                        for (int c = v0 + lane; c < v1; c += 32) {
                            uint4 p[GR];
#pragma unroll
                            for (int j = 0; j < GR; ++j) p[j] = w[j * nv + c];
#pragma unroll
                            for (int m = 0; m < MR; ++m) {
                                const float4 lo = *reinterpret_cast<const float4 *>(xs + m * K8 + c * 4), hi = *reinterpret_cast<const float4 *>(xs + m * K8 + half + c * 4);
#pragma unroll
                                for (int j = 0; j < GR; ++j) acc[m][j0 + j] = mvd_dot8(p[j], lo, hi, acc[m][j0 + j]);
                            }
                        }
                    }
                    __syncwarp();
                    if (lane == 0) skn_mbar_arrive(&empty_bar[s]);
                    if (++s == stages) {
                        s = 0;
                        phase ^= 1u;
                        w = reinterpret_cast<const uint4 *>(ring);
                    } else {
                        w += GR * nv;
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < MR; ++m) {
#pragma unroll
                for (int o = 16, n = 4; o >= 4; o >>= 1, n >>= 1)
#pragma unroll
                    for (int j = 0; j < n; ++j) {
                        const bool up = lane & o;
                        const float mine = up ? acc[m][j + n] : acc[m][j], other = up ? acc[m][j] : acc[m][j + n];
                        acc[m][j] = mine + __shfl_xor_sync(0xffffffffu, other, o);
                    }
                float t = acc[m][0];
                t += __shfl_xor_sync(0xffffffffu, t, 2);
                t += __shfl_xor_sync(0xffffffffu, t, 1);
                if ((lane & 3) == 0) {
                    float *p = &part[buf][m][warp][filled + mvd_row(lane)];
                    *p = pc > 0 ? *p + t : t * rs[m];
                }
            }
            filled += rows;
            if (last && (filled + 8 > MVD_ROWS || g0 + 8 >= r1 - r0)) {
                mvd_barrier();
                auto total = [&](int m, int r) {
                    float t = 0.f;
#pragma unroll
                    for (int w8 = 0; w8 < MVD_WARPS; ++w8) t += part[buf][m][w8][r];
                    return t;
                };
                if constexpr (PAIRS) {
                    const int np = (filled + 1) / 2;
                    for (int j = threadIdx.x; j < np * MR; j += MVD_WARPS * 32) {
                        const int m = j / np, r = j % np * 2;
                        const bool both = r + 1 < filled;
                        const float a = total(m, r), b = both ? total(m, r + 1) : 0.f;
                        dense_store_pair<SKN_EPI_SILU_TAIL>(e, m0 + m, base + r, a, b, both);
                    }
                } else for (int j = threadIdx.x; j < filled * MR; j += MVD_WARPS * 32) {
                    const int m = j / filled, r = j % filled;
                    dense_store_any(e, m0 + m, base + r, total(m, r));
                }
                base += filled;
                filled = 0;
                buf ^= 1;                              // the other half is free: every warp has passed the barrier of its readers
            }
        }
        if (!last) mvd_barrier();                      // (the sums of squares are written again)
    }
}

// vectors per lane of a row of `cols` columns
static int mvd_uu(int64_t cols) { return (int)(((cols / 8 + MVD_WARPS - 1) / MVD_WARPS + 31) / 32); }
constexpr int MVD_MAX_UU = 7;
constexpr int64_t MVD_PIECE = (int64_t)MVD_MAX_UU * 32 * MVD_WARPS * 8;      // columns of x that the registers hold

template <int MR, int UU, int PICK, bool PAIRS, bool EXT>
static cudaError_t launch_mvd_kernel(skn_ctx *ctx, const skn_linear &l, int pieces, int64_t pitch, int m0, cudaStream_t st) {
    auto kern = skn_dense_matvec_kernel<MR, UU, PICK, PAIRS, EXT>;
    static bool attr_done[64] = {false};
    if (!attr_done[ctx->device & 63]) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, mvd_smem(MR));
        if (e != cudaSuccess) return e;
        attr_done[ctx->device & 63] = true;
    }
    const int N = PICK == SKN_PICK_ROWS ? l.pick.n * l.pick.rows_per : (int)l.w->n_rows, K = (int)skn_linear_cols(l), rows = mvd_stage_rows(MR, UU);
    const int64_t row_bytes = PICK == SKN_PICK_COLS ? K * (int64_t)2 : l.w->pitch;
    const size_t xbytes = UU > 0 ? 0 : (size_t)MR * pitch * 2;
    size_t room = mvd_smem(MR) - xbytes;
    if (room > (size_t)MVD_RING) room = MVD_RING;
    int stages = (int)(room / (rows * pitch));
    if (stages < 1) return cudaErrorNotSupported;
    if (stages > MVD_MAX_STAGES) stages = MVD_MAX_STAGES;
    const int units = PAIRS ? (N + 1) / 2 : N;
    const int grid = units < ctx->sm_count ? units : ctx->sm_count;
    const mvd_norm nm = {l.gain, l.eps, l.gain ? l.norm_cols : 0, l.norm_parts > 0 ? l.norm_parts : 1};
    const mvd_pick pk = {l.pick.expert, PICK == SKN_PICK_COLS ? (const uint8_t *)l.pick.w2->d_blocks : nullptr, l.w->pitch,
                         PICK == SKN_PICK_COLS ? l.pick.w2->pitch : 0, l.pick.n, l.pick.rows_per};
    return skn_launch_pdl(kern, dim3(grid), dim3(MVD_THREADS), (size_t)stages * rows * pitch + xbytes, st, 1, (const uint8_t *)l.w->d_blocks, l.w->pitch,
                          row_bytes, pieces, pitch, N, K, m0, l.x32, l.ld_x32, l.x32b, l.ld_x32b, l.x32b ? (int)l.k_a : K, nm, pk, stages, l.epi, ctx->d_status);
}

template <int MR, int UU, int PICK>
static cudaError_t launch_mvd(skn_ctx *ctx, const skn_linear &l, int pieces, int64_t pitch, int m0, cudaStream_t st) {
    const bool pairs = l.epi.kind == SKN_EPI_SILU_TAIL;
    if constexpr (PICK != SKN_PICK_COLS)
        if (pairs) return launch_mvd_kernel<MR, UU, PICK, true, false>(ctx, l, 1, pitch, m0, st);
    if (pairs) return cudaErrorInvalidValue;
    if constexpr (PICK == SKN_PICK_ROWS) return cudaErrorInvalidValue;
    else {
        if (PICK == SKN_PICK_COLS || pieces > 1 || (l.gain && l.norm_cols > 0)) return launch_mvd_kernel<MR, UU, PICK, false, true>(ctx, l, pieces, pitch, m0, st);
        if constexpr (PICK == SKN_PICK_NONE) return launch_mvd_kernel<MR, UU, PICK, false, false>(ctx, l, 1, pitch, m0, st);
        return cudaErrorInvalidValue;
    }
}

// one activation row; more columns than the registers hold go in pieces where the kernel can (the norm within the first one, few rows per CTA)
template <int PICK>
static cudaError_t launch_mvd_row(skn_ctx *ctx, const skn_linear &l, int64_t cols, int m0, cudaStream_t st) {
    int pieces = 1;
    int64_t size = cols;
    if (cols > MVD_PIECE && PICK != SKN_PICK_ROWS && !skn_epi_pairs(l.epi.kind) && (!l.gain || (l.norm_cols > 0 && l.norm_cols <= MVD_PIECE)) &&
        (l.w->n_rows + ctx->sm_count - 1) / ctx->sm_count <= MVD_ROWS - 8) {
        pieces = (int)((cols + MVD_PIECE - 1) / MVD_PIECE);
        size = ((cols + pieces - 1) / pieces + 7) / 8 * 8;
        if (l.gain && size < l.norm_cols) size = l.norm_cols;
        pieces = (int)((cols + size - 1) / size);
    }
    switch (mvd_uu(size)) {
    case 1: return launch_mvd<1, 1, PICK>(ctx, l, pieces, size * 2, m0, st);
    case 2: return launch_mvd<1, 2, PICK>(ctx, l, pieces, size * 2, m0, st);
    case 3: return launch_mvd<1, 3, PICK>(ctx, l, pieces, size * 2, m0, st);
    case 4: return launch_mvd<1, 4, PICK>(ctx, l, pieces, size * 2, m0, st);
    case 5: return launch_mvd<1, 5, PICK>(ctx, l, pieces, size * 2, m0, st);
    case 6: return launch_mvd<1, 6, PICK>(ctx, l, pieces, size * 2, m0, st);
    case 7: return launch_mvd<1, 7, PICK>(ctx, l, pieces, size * 2, m0, st);
    default: return launch_mvd<1, 0, PICK>(ctx, l, 1, cols * 2, m0, st);
    }
}

cudaError_t skn_launch_dense_matvec(skn_ctx *ctx, const skn_linear &l, cudaStream_t st) {
    const int64_t cols = l.pick.kind == SKN_PICK_COLS ? skn_linear_cols(l) : l.w->pitch / 2, pitch = cols * 2;
    if (l.gain && l.norm_cols > 0 && !skn_norm_folds(l.norm_cols, l.norm_parts)) return cudaErrorInvalidValue;
    if ((l.pick.kind && l.M != 1) || l.epi.kind == SKN_EPI_ROTATE) return cudaErrorInvalidValue;
    if (l.pick.kind == SKN_PICK_ROWS) return launch_mvd_row<SKN_PICK_ROWS>(ctx, l, cols, 0, st);
    if (l.pick.kind == SKN_PICK_COLS) return launch_mvd_row<SKN_PICK_COLS>(ctx, l, cols, 0, st);
    if (pitch * 3 > mvd_smem(1)) return cudaErrorNotSupported;       // one stage and one activation row must fit
    for (int m0 = 0; m0 < l.M;) {
        const int left = l.M - m0;
        cudaError_t e;
        int mr = 1;
        if (left >= 4 && pitch * 10 <= mvd_smem(4)) { mr = 4; e = launch_mvd<4, 0, SKN_PICK_NONE>(ctx, l, 1, pitch, m0, st); }
        else if (left >= 2 && pitch * 6 <= mvd_smem(2)) { mr = 2; e = launch_mvd<2, 0, SKN_PICK_NONE>(ctx, l, 1, pitch, m0, st); }
        else e = launch_mvd_row<SKN_PICK_NONE>(ctx, l, cols, m0, st);
        if (e != cudaSuccess) return e;
        m0 += mr;
    }
    return cudaSuccess;
}

// ---- fp32 ----------------------------------------------------------------------------------------------------
// 64 tokens x 64 weight rows per CTA, K in steps of 16; a thread owns 4 x 4 outputs
constexpr int F32_BM = 64, F32_BN = 64, F32_BK = 16;

template <int EPI, bool GROUPS>
__global__ void __launch_bounds__(256)
skn_dense_f32_kernel(const uint8_t *__restrict__ W, int64_t pitch, int N, int K, int M, const float *__restrict__ x, int64_t ldx,
                     const float *__restrict__ xb, int64_t ldxb, int ka, const int32_t *offset, int E, skn_epi e) {
    __shared__ float xt[F32_BK][F32_BM + 4], wt[F32_BK][F32_BN + 4];
    __shared__ int start[GROUPS ? SKN_MAX_EXPERTS + 1 : 1], off[GROUPS ? SKN_MAX_EXPERTS + 1 : 1];
    const int n0 = blockIdx.x * F32_BN;
    int m0 = blockIdx.y * F32_BM;
    const int tm = (threadIdx.x >> 4) * 4, tn = (threadIdx.x & 15) * 4;
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    if (GROUPS) {
        if (threadIdx.x < 32) dense_group_tiles(offset, E, F32_BM, start, off);
        __syncthreads();
        if ((int)blockIdx.y >= start[E]) return;
        const int g = dense_group_of(start, E, blockIdx.y);
        m0 = off[g] + ((int)blockIdx.y - start[g]) * F32_BM;
        M = off[g + 1];
        W += (int64_t)g * N * pitch;
    }
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
        for (int j = 0; j < 4; j += skn_epi_pairs(EPI) ? 2 : 1) {
            if (m0 + tm + i >= M || n0 + tn + j >= N) continue;
            if constexpr (skn_epi_pairs(EPI)) dense_store_pair<EPI>(e, m0 + tm + i, n0 + tn + j, acc[i][j], acc[i][j + 1], n0 + tn + j + 1 < N);
            else dense_store<EPI>(e, m0 + tm + i, n0 + tn + j, acc[i][j]);
        }
}

// most tiles of T rows that M rows in E groups can need
static int group_tiles_bound(int M, int E, int T) { return (M + T - 1) / T + (E < M ? E : M); }

template <int EPI>
static cudaError_t launch_f32(const skn_linear &l, cudaStream_t st) {
    const bool groups = l.pick.kind == SKN_PICK_GROUPS;
    const int N = groups ? l.pick.rows_per : (int)l.w->n_rows, K = (int)l.w->n_cols;
    const dim3 grid((N + F32_BN - 1) / F32_BN, groups ? group_tiles_bound(l.M, l.pick.n, F32_BM) : (l.M + F32_BM - 1) / F32_BM);
    const int ka = l.x32b ? (int)l.k_a : K;
    if constexpr (EPI == SKN_EPI_STORE || EPI == SKN_EPI_SILU_TAIL)
        if (groups)
            return skn_launch_pdl(skn_dense_f32_kernel<EPI, true>, grid, dim3(256), 0, st, 1, (const uint8_t *)l.w->d_blocks, l.w->pitch, N, K, l.M,
                                  l.x32, l.ld_x32, l.x32b, l.ld_x32b, ka, l.pick.offset, l.pick.n, l.epi);
    if (groups) return cudaErrorInvalidValue;
    return skn_launch_pdl(skn_dense_f32_kernel<EPI, false>, grid, dim3(256), 0, st, 1, (const uint8_t *)l.w->d_blocks, l.w->pitch, N, K, l.M,
                          l.x32, l.ld_x32, l.x32b, l.ld_x32b, ka, (const int32_t *)nullptr, 0, l.epi);
}

cudaError_t skn_launch_dense_f32(skn_ctx *, const skn_linear &l, cudaStream_t st) {
    if (l.M == 0) return cudaSuccess;
    switch (l.epi.kind) {
    case SKN_EPI_STORE: return launch_f32<SKN_EPI_STORE>(l, st);
    case SKN_EPI_ADD: return launch_f32<SKN_EPI_ADD>(l, st);
    case SKN_EPI_RELU2: return launch_f32<SKN_EPI_RELU2>(l, st);
    case SKN_EPI_GELU_TABLE: return launch_f32<SKN_EPI_GELU_TABLE>(l, st);
    case SKN_EPI_GELU_TAIL: return launch_f32<SKN_EPI_GELU_TAIL>(l, st);
    case SKN_EPI_SILU_TAIL: return launch_f32<SKN_EPI_SILU_TAIL>(l, st);
    case SKN_EPI_ROTATE: return launch_f32<SKN_EPI_ROTATE>(l, st);
    }
    return cudaErrorInvalidValue;
}

// ---- tensor cores ------------------------------------------------------------------------------------------------
constexpr int DTC_BM = 128, DTC_BK = 64;
constexpr int DTC_A_BYTES = DTC_BM * DTC_BK * 2;
constexpr int DTC_EPI = 8, DTC_MMA = DTC_EPI, DTC_TMA = DTC_EPI + 1;   // eight epilogue warps (two per quarter of TMEM's lanes), MMA, TMA
constexpr int DTC_THREADS = (DTC_EPI + 2) * 32;
constexpr int DTC_GROUP_BOX = 64;                // tokens of one TMA box of a grouped tile
constexpr int DTC_SMEM = 208 * 1024;
constexpr int DTC_MAX_STAGES = 8;

__device__ __forceinline__ void dtc_barrier_epilogue() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

struct dtc_tile {
    int m0, cols, sp, n0, w0;           // first token and tokens of the tile, K split, first row of the output, and of the weight
};

template <int EPI, bool GROUPS>
__global__ void __launch_bounds__(DTC_THREADS, 1)
skn_dense_tc_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x, int N, int K, int M, int NT,
                    int stages, int splits, float *__restrict__ partial, unsigned *__restrict__ tickets, const int32_t *offset, int E, skn_epi e,
                    int32_t *__restrict__ status) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ uint64_t full_bar[DTC_MAX_STAGES], empty_bar[DTC_MAX_STAGES], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_slot, last_flag;
    __shared__ int start[GROUPS ? SKN_MAX_EXPERTS + 1 : 1], off[GROUPS ? SKN_MAX_EXPERTS + 1 : 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int stage_bytes = DTC_A_BYTES + NT * DTC_BK * 2;
    const int acc_cols = NT < 32 ? 32 : NT;
    uint32_t tmem_cols = 32;
    while ((int)tmem_cols < 2 * acc_cols) tmem_cols *= 2;
    const int ksteps = (K + DTC_BK - 1) / DTC_BK;
    const int nt = (N + DTC_BM - 1) / DTC_BM;
    int mt = (M + NT - 1) / NT, units = mt * nt * splits;      // token tiles fastest, then splits, then weight tiles
    auto tile_of = [&](int u) {
        dtc_tile t;
        t.sp = GROUPS ? 0 : (u / mt) % splits;
        t.n0 = (u / mt / splits) * DTC_BM;
        t.w0 = t.n0;
        t.m0 = (u % mt) * NT;
        t.cols = min(NT, M - t.m0);
        if (GROUPS) {
            // a group's tiles are of one size
            const int g = dense_group_of(start, E, u % mt), n = start[g + 1] - start[g], size = ((off[g + 1] - off[g] + n - 1) / n + 15) / 16 * 16;
            t.m0 = off[g] + (u % mt - start[g]) * size;
            t.cols = min(size, off[g + 1] - t.m0);
            t.w0 += g * N;
        }
        return t;
    };

    if (threadIdx.x == 0) {
        for (int s = 0; s < stages; ++s) {
            skn_mbar_init(&full_bar[s], 1);
            skn_mbar_init(&empty_bar[s], 1);
        }
        for (int b = 0; b < 2; ++b) {
            skn_mbar_init(&acc_full[b], 1);
            skn_mbar_init(&acc_empty[b], DTC_EPI);
        }
        skn_fence_mbar_init();
    }
    if (warp == DTC_MMA) tc_alloc(&tmem_slot, tmem_cols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    // the weights depend on no kernel before this one: the first unit's first stages are requested ahead of the wait
    int early = 0;
    if (!GROUPS && warp == DTC_TMA && lane == 0 && (int)blockIdx.x < units) {
        const int sp = (blockIdx.x / mt) % splits, n0 = (blockIdx.x / mt / splits) * DTC_BM;
        const int kb = (int)((int64_t)ksteps * sp / splits), ke = (int)((int64_t)ksteps * (sp + 1) / splits);
        for (; early < stages && early < ke - kb; ++early) {
            skn_mbar_expect_tx(&full_bar[early], (uint32_t)stage_bytes);
            tc_tma_load_2d(smem + (size_t)early * stage_bytes, &tmap_w, (kb + early) * DTC_BK, n0, &full_bar[early]);
        }
    }
    skn_pdl_wait();
    if (GROUPS) {
        if (warp == 0) dense_group_tiles(offset, E, NT, start, off);
        __syncthreads();
        mt = start[E];
        units = mt * nt;
    }

    if (warp == DTC_TMA) {
        if (lane == 0) {
            bool ok = true;
            int it = 0;
            for (int u = blockIdx.x; u < units && ok; u += gridDim.x) {
                const dtc_tile tl = tile_of(u);
                const int m0 = tl.m0, sp = tl.sp, n0 = tl.w0;
                const int kb = (int)((int64_t)ksteps * sp / splits), ke = (int)((int64_t)ksteps * (sp + 1) / splits);
                for (int k = kb; k < ke; ++k, ++it) {
                    const int s = it % stages;
                    uint8_t *a = smem + (size_t)s * stage_bytes;
                    if (it >= early) {
                        if (!skn_mbar_wait(&empty_bar[s], ((uint32_t)(it / stages) & 1u) ^ 1u)) {
                            atomicExch(status, SKN_ERR_TIMEOUT);
                            ok = false;
                            break;
                        }
                        const int boxes = (tl.cols + DTC_GROUP_BOX - 1) / DTC_GROUP_BOX, box = min(NT, DTC_GROUP_BOX);
                        skn_mbar_expect_tx(&full_bar[s], (uint32_t)(GROUPS ? DTC_A_BYTES + boxes * box * DTC_BK * 2 : stage_bytes));
                        tc_tma_load_2d(a, &tmap_w, k * DTC_BK, n0, &full_bar[s]);
                        if (GROUPS)
                            for (int x = 0; x < boxes; ++x) tc_tma_load_2d(a + DTC_A_BYTES + x * box * DTC_BK * 2, &tmap_x, k * DTC_BK, m0 + x * box, &full_bar[s]);
                    }
                    if (!GROUPS) tc_tma_load_2d(a + DTC_A_BYTES, &tmap_x, k * DTC_BK, m0, &full_bar[s]);
                }
            }
            skn_pdl_launch_dependents();           // every load of this CTA is on its way: the next launch may come in
            // the last copies have landed before this CTA ends: drain the stages still in flight
            for (int j = it > stages ? it - stages : 0; j < it && ok; ++j)
                if (!skn_mbar_wait(&full_bar[j % stages], (uint32_t)(j / stages) & 1u)) {
                    atomicExch(status, SKN_ERR_TIMEOUT);
                    ok = false;
                }
        }
    } else if (warp == DTC_MMA) {
        if (lane == 0) {
            uint32_t idesc = tc_idesc(DTC_BM, NT);
            bool ok = true;
            int it = 0, tile = 0;
            for (int u = blockIdx.x; u < units && ok; u += gridDim.x, ++tile) {
                const int sp = GROUPS ? 0 : (u / mt) % splits;
                const int kb = (int)((int64_t)ksteps * sp / splits), ke = (int)((int64_t)ksteps * (sp + 1) / splits);
                const int b = tile & 1;
                if (GROUPS) idesc = tc_idesc(DTC_BM, max(16, (tile_of(u).cols + 15) / 16 * 16));
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
            const dtc_tile tl = tile_of(u);
            const int m0 = tl.m0, sp = tl.sp, nti = u / mt / splits, n0 = tl.n0;
            const int b = tile & 1;
            if (ok && !skn_mbar_wait(&acc_full[b], (uint32_t)(tile >> 1) & 1u)) {
                if (lane == 0) atomicExch(status, SKN_ERR_TIMEOUT);
                ok = false;
            }
            tc_fence_after();
            const int quarter = warp & 3, second = warp >> 2;       // the two warps of a quarter take turns by 32 tokens
            const int n = n0 + quarter * 32 + lane;
            const int cols = tl.cols;
            const uint32_t src = tmem + (uint32_t)(b * acc_cols) + ((uint32_t)(quarter * 32) << 16);
            const int tidx = nti * mt + u % mt;
            float *pbase = partial + ((size_t)tidx * splits) * NT * DTC_BM + quarter * 32 + lane;
#pragma unroll 1
            for (int c0 = second * 32; c0 < cols; c0 += 64) {
                uint32_t acc[32];
                tc_ld32(src + c0, acc);
                if (splits == 1) {
                    float v[32];
#pragma unroll
                    for (int c = 0; c < 32; ++c) v[c] = __uint_as_float(acc[c]);
                    dense_store_warp<EPI, 32>(e, N, m0 + c0, n, v, cols - c0, ok);
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
                    for (int c0 = second * 16; c0 < cols; c0 += 32) {
                        float v[16];
#pragma unroll
                        for (int c = 0; c < 16; ++c) v[c] = 0.f;
#pragma unroll 2
                        for (int s = 0; s < splits; ++s)
#pragma unroll
                            for (int c = 0; c < 16; ++c) v[c] += __ldcg(pbase + ((size_t)s * NT + c0 + c) * DTC_BM);
                        dense_store_warp<EPI, 16>(e, N, m0 + c0, n, v, cols - c0, ok);
                    }
                    if (threadIdx.x == 0) tickets[tidx] = 0;
                }
                dtc_barrier_epilogue();
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == DTC_MMA) {
        __syncwarp();
        tc_fence_after();
        tc_dealloc(tmem, tmem_cols);
    }
}

template <int EPI, bool GROUPS>
static cudaError_t launch_dtc(skn_ctx *ctx, const skn_linear &l, const skn_dense_ws &ws, cudaStream_t st) {
    auto kern = skn_dense_tc_kernel<EPI, GROUPS>;
    static bool attr_done[64] = {false};
    if (!attr_done[ctx->device & 63]) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, DTC_SMEM + 1024);
        if (e != cudaSuccess) return e;
        attr_done[ctx->device & 63] = true;
    }
    const int N = GROUPS ? l.pick.rows_per : (int)l.w->n_rows, K = (int)l.w->n_cols, M = l.M, sms = ctx->sm_count;
    const int nt = (N + DTC_BM - 1) / DTC_BM;
    const int ksteps = (K + DTC_BK - 1) / DTC_BK;
    // token tile: the narrowest that covers M; beyond that, of the widths whose operands the shared memory feeds at full
    // rate, the one with the least time in waves (a wave of narrower tiles costs less, but loads more per product)
    int NT = 16;
    if (GROUPS) {
        // tiles that an expert's share of the rows fills about once
        while (NT < 256 && NT * l.pick.n < M + M / 4) NT *= 2;
    } else if (M <= 128) {
        while (NT < M) NT *= 2;
    } else {
        const int width[3] = {256, 192, 128};
        const double rate[3] = {1.0, 1.03, 1.12};
        double best = 1e30;
        for (int i = 0; i < 3; ++i) {
            const int64_t tiles = (int64_t)nt * ((M + width[i] - 1) / width[i]);
            const double cost = (double)((tiles + sms - 1) / sms) * (width[i] + 8) * rate[i];
            if (cost < best) {
                best = cost;
                NT = width[i];
            }
        }
    }
    while (!GROUPS && NT > 32 && nt * ((M + NT - 1) / NT) * 2 <= sms) NT = NT == 192 ? 128 : NT / 2;
    const int mt = GROUPS ? group_tiles_bound(M, l.pick.n, NT) : (M + NT - 1) / NT;
    // K splits that even out the load of the SMs (the tiles of a decode-size step are fewer than the SMs, or not many more)
    int splits = 1;
    if (!GROUPS && mt * nt < 2 * sms && mt * nt <= SKN_DENSE_MAX_TILES) {
        double best = 1e30;
        for (int s = 1; s <= 16 && (s == 1 || s <= ksteps / 4); ++s) {
            if (s > 1 && (size_t)mt * nt * s * NT * DTC_BM > SKN_DENSE_WS_FLOATS) break;
            const int64_t waves = ((int64_t)mt * nt * s + sms - 1) / sms;
            // per unit: its K steps, a fixed cost, and the partial sums that go out and come back
            const double cost = waves * ((double)ksteps / s + 2.0 + (s > 1 ? NT / 16.0 : 0.0)) + (s > 1 ? s * NT / 32.0 : 0.0);
            if (cost < best * 0.97) {
                best = cost;
                splits = s;
            }
        }
    }
    const int stage_bytes = DTC_A_BYTES + NT * DTC_BK * 2;
    // narrow tiles leave room for the CTA of the next launch, which then requests its weights early
    int stages = (NT <= 64 ? DTC_SMEM / 2 : DTC_SMEM) / stage_bytes;
    if (stages > DTC_MAX_STAGES) stages = DTC_MAX_STAGES;
    CUtensorMap tw, tx;
    cudaError_t e = skn_tmap_bf16(l.w->d_blocks, l.w->n_rows, K, l.w->pitch, DTC_BM, &tw);
    if (e == cudaSuccess) e = skn_tmap_bf16(l.x16, M, K, l.ld_x16 * 2, GROUPS && NT > DTC_GROUP_BOX ? DTC_GROUP_BOX : NT, &tx);
    if (e != cudaSuccess) return e;
    const int units = mt * nt * splits;
    return skn_launch_pdl(kern, dim3(units < sms ? units : sms), dim3(DTC_THREADS), (size_t)stages * stage_bytes + 1024, st, 1, tw, tx, N, K, M, NT,
                          stages, splits, ws.partial, ws.tickets, l.pick.offset, l.pick.n, l.epi, ctx->d_status);
}

cudaError_t skn_launch_dense_tc(skn_ctx *ctx, const skn_linear &l, const skn_dense_ws &ws, cudaStream_t st) {
    if (l.ld_x16 % 8) return cudaErrorInvalidValue;
    if (l.M == 0) return cudaSuccess;
    if (l.pick.kind == SKN_PICK_GROUPS) {
        if (l.epi.kind == SKN_EPI_STORE) return launch_dtc<SKN_EPI_STORE, true>(ctx, l, ws, st);
        if (l.epi.kind == SKN_EPI_SILU_TAIL) return launch_dtc<SKN_EPI_SILU_TAIL, true>(ctx, l, ws, st);
        return cudaErrorInvalidValue;
    }
    switch (l.epi.kind) {
    case SKN_EPI_STORE: return launch_dtc<SKN_EPI_STORE, false>(ctx, l, ws, st);
    case SKN_EPI_ADD: return launch_dtc<SKN_EPI_ADD, false>(ctx, l, ws, st);
    case SKN_EPI_RELU2: return launch_dtc<SKN_EPI_RELU2, false>(ctx, l, ws, st);
    case SKN_EPI_GELU_TABLE: return launch_dtc<SKN_EPI_GELU_TABLE, false>(ctx, l, ws, st);
    case SKN_EPI_GELU_TAIL: return launch_dtc<SKN_EPI_GELU_TAIL, false>(ctx, l, ws, st);
    case SKN_EPI_SILU_TAIL: return launch_dtc<SKN_EPI_SILU_TAIL, false>(ctx, l, ws, st);
    case SKN_EPI_ROTATE: return launch_dtc<SKN_EPI_ROTATE, false>(ctx, l, ws, st);
    }
    return cudaErrorInvalidValue;
}
