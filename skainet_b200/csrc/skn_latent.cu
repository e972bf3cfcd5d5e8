// Latent attention (see skn_latent.cuh).
#include "skn_latent.cuh"
#include "skn_mma.cuh"

#include <algorithm>
#include <math.h>

constexpr int LT = 256;                  // threads
constexpr int QL_COLS = 128;             // latent columns of a CTA of the absorbed query kernel
constexpr int OL_ROWS = 32;              // value rows of a CTA of the absorbed output kernel
constexpr int LA_MAX_SPLITS = 320;       // key splits of a query row; at most LA_TARGET CTAs beyond one per (row, head group) are asked for
constexpr int LA_TARGET = 296;

__device__ __forceinline__ float lat_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float lat_sum(float v, float *red) {
    v = lat_warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (int w = 0; w < (int)(blockDim.x >> 5); ++w) t += red[w];
    __syncthreads();
    return t;
}
__device__ __forceinline__ void lat_unpack(const uint4 &v, float (&o)[8]) {
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        o[2 * i] = __uint_as_float(w[i] << 16);
        o[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
    }
}
// element d of a rotated part: the pair (d & ~1, d | 1) turned by the row's angle
__device__ __forceinline__ float lat_turn(const float *src, int d, const skn_rot &rot, int64_t m) {
    const float v = __ldcg(src + d);
    if ((d >> 1) >= rot.half) return v;
    const float2 cs = __ldcg(rot.table + m * rot.ld + (d >> 1));
    const float o = __ldcg(src + (d ^ 1));
    return (d & 1) ? v * cs.x + o * cs.y : v * cs.x - o * cs.y;
}
__device__ __forceinline__ void lat_store(float *p, float v) { *p = v; }
__device__ __forceinline__ void lat_store(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }

// the CTA files row m's latent and rotated key
template <class CT>
__device__ __forceinline__ void lat_append(const skn_latent_args &a, const skn_step &st, CT *kc, int cap, int pitch, int m, float *red) {
    const int slot = st.slot0 + m / st.T, pos = min(st.pos[slot] + m % st.T, st.max_pos - 1);
    CT *dst = kc + ((int64_t)slot * cap + pos % cap) * pitch;
    const float *src = a.dkv + m * a.ld;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.kv_rank; i += LT) {
        const float v = __ldcg(src + i);
        ss = fmaf(v, v, ss);
    }
    const float r = 1.f / sqrtf(lat_sum(ss, red) / (float)a.kv_rank + a.eps);
    for (int i = threadIdx.x; i < a.kv_rank; i += LT) lat_store(dst + i, __ldcg(src + i) * r * __ldg(a.kv_gain + i));
    for (int i = threadIdx.x; i < a.rp; i += LT) lat_store(dst + a.kvp + i, lat_turn(src + a.kvp, i, a.rot, m));
}

template <class CT>
__global__ void __launch_bounds__(LT)
skn_latent_rows_kernel(skn_latent_args a, skn_step st, CT *kc, int cap, int pitch, skn_rows_out cq) {
    __shared__ float red[LT / 32];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int64_t m = blockIdx.x;
    lat_append(a, st, kc, cap, pitch, (int)m, red);
    if (!cq.y32 && !cq.y16) return;
    const float *src = a.dq + m * a.ld;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.q_rank; i += LT) {
        const float v = __ldcg(src + i);
        ss = fmaf(v, v, ss);
    }
    const float r = 1.f / sqrtf(lat_sum(ss, red) / (float)a.q_rank + a.eps);
    for (int i = threadIdx.x; i < a.q_rank; i += LT) {
        const float v = __ldcg(src + i) * r * __ldg(a.q_gain + i);
        if (cq.y32) cq.y32[m * cq.ld32 + i] = v;
        if (cq.y16) cq.y16[m * cq.ld16 + i] = __float2bfloat16_rn(v);
    }
}

cudaError_t skn_launch_latent_rows(const skn_step &s, const skn_latent_args &a, const skn_rows_out &cq, cudaStream_t st) {
    const dim3 grid(s.n_seqs * s.T);
    if (a.kv->dtype == SKN_KV_BF16)
        return skn_launch_pdl(skn_latent_rows_kernel<__nv_bfloat16>, grid, dim3(LT), 0, st, 1, a, s, (__nv_bfloat16 *)a.kv->d_k, a.kv->capacity, a.kv->k_pitch, cq);
    return skn_launch_pdl(skn_latent_rows_kernel<float>, grid, dim3(LT), 0, st, 1, a, s, (float *)a.kv->d_k, a.kv->capacity, a.kv->k_pitch, cq);
}

// ---- absorbed form --------------------------------------------------------------------------------------------------
// ql[m][h] = [W_uk,h^T q_h | rotated q_h].  CTA: QL_COLS latent columns of one head, RB rows; thread: eight columns, every 16th dimension.
// With APPEND, CTAs from `tiles` on (one per row of the step, spread over the z dimension) file the newest latents, the last one routes.
// smem (floats): q [RB][dim] | sums [16][RB][QL_COLS]
template <class CT, int RB>
__global__ void __launch_bounds__(LT)
skn_latent_q_kernel(skn_latent_args a, skn_step st, CT *kc, int cap, int pitch, const uint8_t *__restrict__ ukv, int64_t wpitch, int tiles, int col_tiles, int M) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[LT / 32];
    const int tid = threadIdx.x, m0 = blockIdx.y * RB, hd = a.dim + a.rp;
    if ((int)blockIdx.x >= tiles) {
        skn_pdl_wait();
        if ((int)blockIdx.x == tiles) {
            for (int m = m0; m < min(M, m0 + RB); ++m) lat_append(a, st, kc, cap, pitch, m, red);
        } else if (tid < 32) {
            for (int m = m0; m < min(M, m0 + RB); ++m) skn_route_row(a.route, m, sm);
        }
        return;
    }
    const int h = blockIdx.x / col_tiles, c0 = (blockIdx.x % col_tiles) * QL_COLS, cv = tid & 15, dg = tid >> 4, c = c0 + cv * 8;
    const uint8_t *w = ukv + (int64_t)h * a.dim * wpitch + (int64_t)c * 2;
    // the weights' way into L2 depends on no kernel before this one
    if (c < a.kvp && (cv & 7) == 0)
        for (int d = dg; d < a.dim; d += 16) asm volatile("prefetch.global.L2 [%0];" ::"l"(w + d * wpitch));
    skn_pdl_wait();
    float *qs = sm, *part = sm + RB * a.dim;
    for (int i = tid; i < RB * a.dim; i += LT) {
        const int r = i / a.dim, d = i % a.dim;
        qs[i] = m0 + r < M ? __ldcg(a.q + ((int64_t)(m0 + r) * a.heads + h) * hd + d) : 0.f;
    }
    __syncthreads();
    float acc[RB][8];
#pragma unroll
    for (int r = 0; r < RB; ++r)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[r][e] = 0.f;
    if (c < a.kvp) {
#pragma unroll 8
        for (int d = dg; d < a.dim; d += 16) {
            float f[8];
            lat_unpack(__ldg(reinterpret_cast<const uint4 *>(w + d * wpitch)), f);
#pragma unroll
            for (int r = 0; r < RB; ++r)
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[r][e] = fmaf(qs[r * a.dim + d], f[e], acc[r][e]);
        }
    }
#pragma unroll
    for (int r = 0; r < RB; ++r)
#pragma unroll
        for (int e = 0; e < 8; ++e) part[(dg * RB + r) * QL_COLS + cv * 8 + e] = acc[r][e];
    __syncthreads();
    const int kd = a.kvp + a.rp;
    for (int i = tid; i < RB * QL_COLS; i += LT) {
        const int r = i / QL_COLS, k = i % QL_COLS;
        if (m0 + r >= M || c0 + k >= a.kvp) continue;
        float t = 0.f;
#pragma unroll
        for (int g = 0; g < 16; ++g) t += part[(g * RB + r) * QL_COLS + k];
        a.ql[((int64_t)(m0 + r) * a.heads + h) * kd + c0 + k] = t;
    }
    if (c0 == 0)
        for (int i = tid; i < RB * a.rp; i += LT) {
            const int r = i / a.rp, d = i % a.rp;
            if (m0 + r >= M) continue;
            const int64_t row = (int64_t)(m0 + r) * a.heads + h;
            a.ql[row * kd + a.kvp + d] = lat_turn(a.q + row * hd + a.dim, d, a.rot, m0 + r);
        }
}

// ---- attention of absorbed queries over a bf16 cache ----------------------------------------------------------------
// CTA: LA_HEADS heads of one query row, `per` tiles of LA_KEYS keys.  The latents are read once for all its heads and serve as keys and as
// values.  Queries and weights enter the tensor cores as two bf16 terms each.  A split leaves its running maximum, sum and weighted
// latents; the output kernel puts the splits together.
constexpr int LA_HEADS = 16, LA_KEYS = 32, LA_PS = LA_KEYS + 8, LA_SS = LA_KEYS + 4;
constexpr float LAT_L2E = 1.4426950408889634f;

// smem: K [2][LA_KEYS][kp + 8] | q, two terms [2][LA_HEADS][kp + 8] | weights, two terms [2][LA_HEADS][LA_PS] (bf16) | scores [4][LA_HEADS][LA_SS] (fp32)
static size_t la_smem(int kp) { return ((size_t)(2 * LA_KEYS + 2 * LA_HEADS) * (kp + 8) + 2 * LA_HEADS * LA_PS) * 2 + (size_t)4 * LA_HEADS * LA_SS * 4; }

__device__ __forceinline__ int lat_first(const skn_latent_args &a, int p) { return a.window > 0 ? max(0, p - a.window + 1) : 0; }

template <int NTW>
__global__ void __launch_bounds__(LT)
skn_latent_attn_kernel(skn_latent_args a, skn_step st, const __nv_bfloat16 *__restrict__ kc, int cap, int kp, int per, int splits, float2 *stats, float *sums) {
    extern __shared__ __align__(16) uint8_t smb[];
    __shared__ float s_corr[LA_HEADS];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, split = blockIdx.x, h0 = blockIdx.y * LA_HEADS, m = blockIdx.z;
    const int ks = kp + 8, qd = a.kvp + a.rp;
    __nv_bfloat16 *K = reinterpret_cast<__nv_bfloat16 *>(smb), *Q = K + 2 * LA_KEYS * ks, *P = Q + 2 * LA_HEADS * ks;
    float *Sp = reinterpret_cast<float *>(P + 2 * LA_HEADS * LA_PS);
    const int slot = st.slot0 + m / st.T, p = min(st.pos[slot] + m % st.T, st.max_pos - 1), lo = lat_first(a, p), total = (p - lo) / LA_KEYS + 1;
    const int t0 = split * per, t1 = min(total, t0 + per);
    if (t0 >= t1) {
        skn_pdl_wait();
        return;
    }
    const __nv_bfloat16 *ring = kc + (int64_t)slot * cap * kp;
    const int cr = tid >> 3, cc = tid & 7;           // a key row's pieces go to eight threads
    {
        // the first tile's way into L2 (the newest key is not written yet: it is fetched after the wait)
        const int j = min(lo + t0 * LA_KEYS + cr, p);
        for (int i = cc * 64; i < kp; i += 512) asm volatile("prefetch.global.L2 [%0];" ::"l"(ring + (int64_t)(j % cap) * kp + i));
    }
    skn_pdl_wait();
    auto load_tile = [&](int t, int buf) {
        const int j = lo + t * LA_KEYS + cr;
        const bool in = j <= p;
        const __nv_bfloat16 *src = ring + (int64_t)(j % cap) * kp;
        const uint32_t dst = skn_smem_u32(K + ((size_t)buf * LA_KEYS + cr) * ks);
        for (int c = cc * 8; c < kp; c += 64) cp_async16(dst + c * 2, src + c, in);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_tile(t0, 0);
    for (int i = tid; i < LA_HEADS * (kp / 2); i += LT) {
        const int r = i / (kp / 2), d = i % (kp / 2) * 2;
        float2 v = make_float2(0.f, 0.f);
        if (h0 + r < a.heads && d < qd) v = __ldcg(reinterpret_cast<const float2 *>(a.ql + ((int64_t)m * a.heads + h0 + r) * qd + d));
        v.x *= a.scale * LAT_L2E;
        v.y *= a.scale * LAT_L2E;
        const uint32_t hi = pack_bf16(v.x, v.y);
        less_bf16(v.x, v.y, hi);
        *reinterpret_cast<uint32_t *>(Q + r * ks + d) = hi;
        *reinterpret_cast<uint32_t *>(Q + (LA_HEADS + r) * ks + d) = pack_bf16(v.x, v.y);
    }
    float o[NTW][2][4];
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int e = 0; e < 8; ++e) o[i][e >> 2][e & 3] = 0.f;
    float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};       // heads 2 warp, 2 warp + 1
    const int sn = warp & 1, sq = warp >> 1, steps = kp / 16, k0 = steps * sq / 4, k1 = steps * (sq + 1) / 4;     // scores: 16 keys, a quarter of the row
    const int tiles = (a.kvp + 15) / 16;
    for (int t = t0; t < t1; ++t) {
        const int buf = (t - t0) & 1;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (t + 1 < t1) load_tile(t + 1, buf ^ 1);
        const __nv_bfloat16 *Kb = K + (size_t)buf * LA_KEYS * ks;
        float s[2][4] = {};
        for (int k = k0; k < k1; ++k) {
            uint32_t ah[4], al[4], bf[4];
            ldsm4(ah, skn_smem_u32(Q + (lane & 15) * ks + k * 16 + (lane >> 4) * 8));
            ldsm4(al, skn_smem_u32(Q + (LA_HEADS + (lane & 15)) * ks + k * 16 + (lane >> 4) * 8));
            ldsm4(bf, skn_smem_u32(Kb + (size_t)(sn * 16 + (lane & 7) + ((lane >> 4) << 3)) * ks + k * 16 + ((lane >> 3) & 1) * 8));
            mma_bf16(s[0], al, bf[0], bf[1]);
            mma_bf16(s[1], al, bf[2], bf[3]);
            mma_bf16(s[0], ah, bf[0], bf[1]);
            mma_bf16(s[1], ah, bf[2], bf[3]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e)
                *reinterpret_cast<float2 *>(Sp + (sq * LA_HEADS + (lane >> 2) + e * 8) * LA_SS + sn * 16 + n * 8 + (lane & 3) * 2) = make_float2(s[n][2 * e], s[n][2 * e + 1]);
        __syncthreads();
        const bool seen = lo + t * LA_KEYS + lane <= p;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int r = warp * 2 + e;
            float v = 0.f;
#pragma unroll
            for (int q = 0; q < 4; ++q) v += Sp[(q * LA_HEADS + r) * LA_SS + lane];
            float mx = seen ? v : -INFINITY;
#pragma unroll
            for (int x = 16; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
            mx = fmaxf(mx, mrow[e]);
            const float w = seen ? exp2f(v - mx) : 0.f, c = exp2f(mrow[e] - mx);
            lrow[e] = lrow[e] * c + lat_warp_sum(w);
            mrow[e] = mx;
            const __nv_bfloat16 hi = __float2bfloat16_rn(w);
            P[r * LA_PS + lane] = hi;
            P[(LA_HEADS + r) * LA_PS + lane] = __float2bfloat16_rn(w - __bfloat162float(hi));
            if (lane == 0) s_corr[r] = c;
        }
        __syncthreads();
        const float c0 = s_corr[lane >> 2], c1 = s_corr[(lane >> 2) + 8];
        uint32_t pf[2][2][4];
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int k = 0; k < 2; ++k) ldsm4(pf[x][k], skn_smem_u32(P + (x * LA_HEADS + (lane & 15)) * LA_PS + k * 16 + (lane >> 4) * 8));
#pragma unroll
        for (int i = 0; i < NTW; ++i) {
            const int n = warp + i * 8;
            if (n >= tiles) continue;
#pragma unroll
            for (int y = 0; y < 2; ++y) {
                o[i][y][0] *= c0; o[i][y][1] *= c0;
                o[i][y][2] *= c1; o[i][y][3] *= c1;
            }
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                uint32_t bf[4];
                ldsm4t(bf, skn_smem_u32(Kb + (size_t)(k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ks + n * 16 + (lane >> 4) * 8));
#pragma unroll
                for (int x = 1; x >= 0; --x) {
                    mma_bf16(o[i][0], pf[x][k], bf[0], bf[1]);
                    mma_bf16(o[i][1], pf[x][k], bf[2], bf[3]);
                }
            }
        }
    }
    skn_pdl_launch_dependents();
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int y = 0; y < 2; ++y)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int h = h0 + (lane >> 2) + e * 8, c = (warp + i * 8) * 16 + y * 8 + (lane & 3) * 2;
                if (h < a.heads && c < a.kvp)
                    *reinterpret_cast<float2 *>(sums + (((int64_t)m * a.heads + h) * splits + split) * a.kvp + c) = make_float2(o[i][y][2 * e], o[i][y][2 * e + 1]);
            }
    if (lane < 2 && h0 + warp * 2 + lane < a.heads)
        stats[((int64_t)m * a.heads + h0 + warp * 2 + lane) * splits + split] = make_float2(lane ? mrow[1] : mrow[0], lane ? lrow[1] : lrow[0]);
}

// out[m][h][v] = sigmoid(gate) * (W_uv row (h, v) . ol[m][h]).  CTA: OL_ROWS rows of one head, RB tokens.  splits > 0: the latents of
// the heads are put together here from the attention's splits, else they are in a.ol.  smem (floats): ol [RB][kvp], as often
// as parts of the splits are summed apart
template <int RB>
__global__ void __launch_bounds__(LT)
skn_latent_out_kernel(skn_latent_args a, skn_step st, const uint8_t *__restrict__ ukv, int64_t wpitch, int row_tiles, int M, int per, int splits,
                      const float2 *stats, const float *sums) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float share[RB][LA_MAX_SPLITS];
    __shared__ int s_live[RB];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, m0 = blockIdx.y * RB;
    const int h = blockIdx.x / row_tiles, v0 = (blockIdx.x % row_tiles) * OL_ROWS, v1 = min(a.vdim, v0 + OL_ROWS);
    const uint8_t *w = ukv + ((int64_t)a.heads * a.dim + (int64_t)h * a.vdim) * wpitch;
    for (int v = v0 + warp; v < v1; v += LT / 32)
        for (int64_t i = (int64_t)lane * 128; i < wpitch; i += 32 * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(w + v * wpitch + i));
    skn_pdl_wait();
    if (splits > 0) {
        // each split's share of the softmax
        if (warp < RB && m0 + warp < M) {
            const int m = m0 + warp, slot = st.slot0 + m / st.T, p = min(st.pos[slot] + m % st.T, st.max_pos - 1);
            const int live = ((p - lat_first(a, p)) / LA_KEYS + per) / per;
            const float2 *rec = stats + ((int64_t)m * a.heads + h) * splits;
            const float sink = a.sink ? a.sink[h] * LAT_L2E : -INFINITY;
            float top = sink, den = 0.f;
            for (int x = lane; x < live; x += 32) top = fmaxf(top, __ldcg(&rec[x].x));
#pragma unroll
            for (int x = 16; x > 0; x >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, x));
            for (int x = lane; x < live; x += 32) den += exp2f(__ldcg(&rec[x].x) - top) * __ldcg(&rec[x].y);
            den = lat_warp_sum(den) + (a.sink ? exp2f(sink - top) : 0.f);
            for (int x = lane; x < live; x += 32) share[warp][x] = exp2f(__ldcg(&rec[x].x) - top) / den;
            if (lane == 0) s_live[warp] = live;
        }
        __syncthreads();
        // a vector of columns by one thread, or its splits by several
        const int vecs = RB * a.kvp / 4, parts = max(1, LT / vecs);
        for (int u = tid; u < vecs * parts; u += LT) {
            const int part = u / vecs, i = (u % vecs) * 4, r = i / a.kvp, k = i % a.kvp;
            float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
            if (m0 + r < M) {
                const float *src = sums + (((int64_t)(m0 + r) * a.heads + h) * splits) * a.kvp + k;
#pragma unroll 8
                for (int x = part; x < s_live[r]; x += parts) {
                    const float4 v = __ldcg(reinterpret_cast<const float4 *>(src + (int64_t)x * a.kvp));
                    const float f = share[r][x];
                    t.x = fmaf(f, v.x, t.x); t.y = fmaf(f, v.y, t.y); t.z = fmaf(f, v.z, t.z); t.w = fmaf(f, v.w, t.w);
                }
            }
            *reinterpret_cast<float4 *>(sm + part * RB * a.kvp + i) = t;
        }
        if (parts > 1) {
            __syncthreads();
            for (int i = tid; i < RB * a.kvp; i += LT) {
                float t = sm[i];
                for (int x = 1; x < parts; ++x) t += sm[x * RB * a.kvp + i];
                sm[i] = t;
            }
        }
    } else {
        for (int i = tid; i < RB * a.kvp; i += LT) {
            const int r = i / a.kvp, k = i % a.kvp;
            sm[i] = m0 + r < M ? __ldcg(a.ol + ((int64_t)(m0 + r) * a.heads + h) * a.kvp + k) : 0.f;
        }
    }
    __syncthreads();
    skn_pdl_launch_dependents();
    constexpr int VR = OL_ROWS / (LT / 32);          // rows of a warp
    float acc[VR][RB];
#pragma unroll
    for (int x = 0; x < VR; ++x)
#pragma unroll
        for (int r = 0; r < RB; ++r) acc[x][r] = 0.f;
    for (int k = lane * 8; k < a.kvp; k += 256) {
#pragma unroll
        for (int x = 0; x < VR; ++x) {
            const int v = v0 + warp + x * (LT / 32);
            if (v >= v1) continue;
            float f[8];
            lat_unpack(__ldg(reinterpret_cast<const uint4 *>(w + v * wpitch + k * 2)), f);
#pragma unroll
            for (int r = 0; r < RB; ++r) {
                const float4 lo = *reinterpret_cast<const float4 *>(sm + r * a.kvp + k), hi = *reinterpret_cast<const float4 *>(sm + r * a.kvp + k + 4);
                acc[x][r] = fmaf(f[0], lo.x, fmaf(f[1], lo.y, fmaf(f[2], lo.z, fmaf(f[3], lo.w, acc[x][r]))));
                acc[x][r] = fmaf(f[4], hi.x, fmaf(f[5], hi.y, fmaf(f[6], hi.z, fmaf(f[7], hi.w, acc[x][r]))));
            }
        }
    }
#pragma unroll
    for (int x = 0; x < VR; ++x)
#pragma unroll
        for (int r = 0; r < RB; ++r) {
            const float t = lat_warp_sum(acc[x][r]);
            const int v = v0 + warp + x * (LT / 32);
            if (lane != 0 || v >= v1 || m0 + r >= M) continue;
            const int64_t m = m0 + r, col = (int64_t)h * a.vdim + v;
            const float o = t / (1.f + expf(-__ldcg(a.gate + m * a.ld + col)));
            if (a.out.y32) a.out.y32[m * a.out.ld32 + col] = o;
            if (a.out.y16) a.out.y16[m * a.out.ld16 + col] = __float2bfloat16_rn(o);
        }
}

template <class CT, int RB>
static cudaError_t launch_q(const skn_step &s, const skn_latent_args &a, bool append, cudaStream_t st) {
    const int M = s.n_seqs * s.T, col_tiles = (a.kvp + QL_COLS - 1) / QL_COLS, tiles = a.heads * col_tiles;
    const bool route = append && a.route.logits;
    const size_t own = ((size_t)RB * a.dim + (size_t)16 * RB * QL_COLS) * sizeof(float), rt = skn_route_smem(a.route);
    return skn_launch_pdl(skn_latent_q_kernel<CT, RB>, dim3(tiles + (append ? 1 : 0) + (route ? 1 : 0), (M + RB - 1) / RB), dim3(LT), own > rt ? own : rt, st, 1, a, s,
                          (CT *)a.kv->d_k, a.kv->capacity, a.kv->k_pitch, (const uint8_t *)a.ukv->d_blocks, a.ukv->pitch, tiles, col_tiles, M);
}

// the split kernel above: a bf16 cache whose rows fit shared memory
static bool tiles_fit(const skn_latent_args &a) { return a.kv->dtype == SKN_KV_BF16 && la_smem(a.kv->k_pitch) <= 220 * 1024; }

template <int NTW>
static cudaError_t launch_la(const skn_step &s, const skn_latent_args &a, int per, int splits, float2 *stats, float *sums, cudaStream_t st) {
    auto kern = skn_latent_attn_kernel<NTW>;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return e;
    return skn_launch_pdl(kern, dim3(splits, (a.heads + LA_HEADS - 1) / LA_HEADS, s.n_seqs * s.T), dim3(LT), la_smem(a.kv->k_pitch), st, 1, a, s,
                          (const __nv_bfloat16 *)a.kv->d_k, a.kv->capacity, a.kv->k_pitch, per, splits, stats, sums);
}

size_t skn_latent_scratch(const skn_latent_args &a, int rows, int max_pos) {
    if (!tiles_fit(a)) return skn_attn_scratch(rows, a.heads, a.kvp, a.window, max_pos);
    // fewer rows may ask for more splits each; the CTAs stay below one per (row, head group) and LA_TARGET more
    const size_t ctas = (size_t)rows * ((a.heads + LA_HEADS - 1) / LA_HEADS) + LA_TARGET;
    return ctas * LA_HEADS * (a.kvp + 2) + 4;
}

cudaError_t skn_launch_latent_absorbed(const skn_step &s, const skn_latent_args &a, bool append, cudaStream_t st) {
    const int M = s.n_seqs * s.T;
    const bool bf = a.kv->dtype == SKN_KV_BF16;
    cudaError_t e = M == 1 ? (bf ? launch_q<__nv_bfloat16, 1>(s, a, append, st) : launch_q<float, 1>(s, a, append, st))
                           : (bf ? launch_q<__nv_bfloat16, 2>(s, a, append, st) : launch_q<float, 2>(s, a, append, st));
    if (e != cudaSuccess) return e;
    const int row_tiles = (a.vdim + OL_ROWS - 1) / OL_ROWS;
    const uint8_t *w = (const uint8_t *)a.ukv->d_blocks;
    int per = 1, splits = 0;
    float2 *stats = nullptr;
    float *sums = nullptr;
    if (tiles_fit(a)) {
        const int groups = (a.heads + LA_HEADS - 1) / LA_HEADS, span = a.window > 0 && a.window < s.max_pos ? a.window : s.max_pos;
        const int tiles = (span + LA_KEYS - 1) / LA_KEYS;
        splits = std::min(tiles, (LA_TARGET + M * groups - 1) / (M * groups));
        per = (tiles + splits - 1) / splits;
        splits = (tiles + per - 1) / per;
        stats = reinterpret_cast<float2 *>(a.scratch);
        sums = a.scratch + ((size_t)M * a.heads * splits * 2 + 3) / 4 * 4;
        const int nt = ((a.kvp + 15) / 16 + 7) / 8;
        e = nt <= 1 ? launch_la<1>(s, a, per, splits, stats, sums, st) : nt <= 2 ? launch_la<2>(s, a, per, splits, stats, sums, st)
            : nt <= 4 ? launch_la<4>(s, a, per, splits, stats, sums, st) : launch_la<8>(s, a, per, splits, stats, sums, st);
    } else {
        // the latents are keys (with the rotated part) and values of one key head
        skn_kvcache view = *a.kv;
        view.d_v = view.d_k;
        view.v_dim = view.v_pitch = a.kvp;
        view.v_stride = view.k_pitch;
        skn_attn_args x = {};
        x.kv = &view; x.heads = a.heads; x.window = a.window; x.scale = a.scale; x.sink = a.sink;
        x.q = a.ql; x.ld = (int64_t)a.heads * (a.kvp + a.rp);
        x.out_scale = 1.f;
        x.out = skn_rows_out{a.ol, (int64_t)a.heads * a.kvp, nullptr, 0};
        x.scratch = a.scratch; x.tickets = a.tickets;
        e = skn_launch_attn_rows(s, x, st);
    }
    if (e != cudaSuccess) return e;
    const int RB = M == 1 ? 1 : 4;
    const size_t osm = std::max((size_t)RB * a.kvp, (size_t)LT * 4) * sizeof(float);
    const dim3 grid(a.heads * row_tiles, (M + RB - 1) / RB);
    if (M == 1) return skn_launch_pdl(skn_latent_out_kernel<1>, grid, dim3(LT), osm, st, 1, a, s, w, a.ukv->pitch, row_tiles, M, per, splits, (const float2 *)stats, (const float *)sums);
    return skn_launch_pdl(skn_latent_out_kernel<4>, grid, dim3(LT), osm, st, 1, a, s, w, a.ukv->pitch, row_tiles, M, per, splits, (const float2 *)stats, (const float *)sums);
}

// ---- expanded form ----------------------------------------------------------------------------------------------------
bool skn_latent_expand_fits(const skn_latent_args &a) { return a.kv->dtype == SKN_KV_BF16 && skn_attn_tiles_fit(a.dim + a.rp, a.vdim); }

cudaError_t skn_launch_latent_expanded(skn_ctx *ctx, const skn_step &s, const skn_latent_args &a, const int32_t *len, const skn_dense_ws &ws, cudaStream_t st) {
    const int64_t ldx = (int64_t)a.heads * (a.dim + a.vdim);
    for (int i = 0; i < s.n_seqs; ++i) {
        const __nv_bfloat16 *ring = (const __nv_bfloat16 *)a.kv->d_k + (int64_t)(s.slot0 + i) * a.kv->capacity * a.kv->k_pitch;
        skn_linear l = {};
        l.w = a.ukv;
        l.M = len[i] < a.kv->capacity ? len[i] : a.kv->capacity;
        l.x16 = ring;
        l.ld_x16 = a.kv->k_pitch;
        l.epi.kind = SKN_EPI_STORE;
        l.epi.y16 = a.kvx;
        l.epi.ld_y16 = ldx;
        cudaError_t e = skn_launch_dense_tc(ctx, l, ws, st);
        if (e != cudaSuccess) return e;
        skn_step one = s;
        one.slot0 += i;
        one.n_seqs = 1;
        const int64_t row = (int64_t)i * s.T;
        skn_attn_args x = {};
        x.heads = a.heads; x.window = a.window; x.scale = a.scale; x.sink = a.sink;
        x.q16 = a.q16 + row * a.heads * (a.dim + a.rp);
        x.out_scale = 1.f;
        x.out = skn_rows_out{a.out.y32 ? a.out.y32 + row * a.out.ld32 : nullptr, a.out.ld32, a.out.y16 ? a.out.y16 + row * a.out.ld16 : nullptr, a.out.ld16};
        x.gate = a.gate + row * a.ld; x.ld_gate = a.ld;
        skn_attn_keys k = {};
        k.kp = a.dim + a.rp; k.k1 = a.dim; k.vp = k.vdim = a.vdim; k.cap = a.kv->capacity; k.group = 1;
        k.k = a.kvx; k.k_row = ldx; k.k_head = a.dim;
        k.k2 = (const __nv_bfloat16 *)a.kv->d_k + a.kvp; k.k2_row = a.kv->k_pitch; k.k2_slot = (int64_t)a.kv->capacity * a.kv->k_pitch;
        k.v = a.kvx + (int64_t)a.heads * a.dim; k.v_row = ldx; k.v_head = a.vdim;
        if ((e = skn_launch_attn_tiles(one, x, k, st)) != cudaSuccess) return e;
    }
    return cudaSuccess;
}

int32_t skn_check_latent_spec(skn_ctx *ctx, const skn_latent_spec *s) {
    if (s->heads < 1 || s->dim < 1 || s->vdim < 1 || s->q_rank < 1 || s->kv_rank < 1 || s->rot_dim < 0 || s->window < 0)
        return skn_fail(ctx, SKN_ERR_ARG, "invalid latent attention geometry");
    if (s->rot_dims < 0 || s->rot_dims % 2 || s->rot_dims > s->rot_dim || s->dim > SKN_ATTN_MAX_DIM || s->vdim > SKN_ATTN_MAX_DIM ||
        s->kv_rank + s->rot_dim + 32 > SKN_KV_MAX_DIM)
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    return SKN_OK;
}
