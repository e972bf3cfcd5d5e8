// Chunked attention and retention (see skn_mixers.cuh).
//
//  skn_mix_decode_kernel   one token per sequence.  Attention CTAs: (128-key split, group of up to four query heads of
//                          one kv head, row); the CTA that holds the newest key normalises, rotates and stores it.
//                          Splits meet in the CTA that draws the last ticket.  Retention CTAs of the same launch: one
//                          head of one row, the state read and written once.
//  skn_head_prep_kernel    many tokens: norm and rotation of every head, K and V into the cache
//  skn_attn_tc_kernel      64 queries of one head: scores and products on the tensor cores (bf16 operands, fp32 sums);
//                          the weights enter the second product as two bf16 terms, so they keep 16 bits
//  skn_attn_rows_kernel    the split kernel on prepared keys (fp32 cache, or head widths beyond the tensor-core form)
//  skn_ret_*_kernel        retention in chunks of 64 tokens: what each chunk adds to the state, the states at the chunk
//                          starts, and the outputs; on the CUDA cores (fp32 decoder) or the tensor cores (two-term tf32)
#include "skn_mixers.cuh"
#include "skn_mma.cuh"

#include <math.h>
#include <stdlib.h>

constexpr int MIX_THREADS = 256;
constexpr int KS = SKN_ATTN_SPLIT_KEYS;

template <class CT> struct CacheVec;
template <> struct CacheVec<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(const float *p, float *o) {
        const float4 v = *reinterpret_cast<const float4 *>(p);
        o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
    }
    static __device__ __forceinline__ float round(float v) { return v; }
    static __device__ __forceinline__ void store(float *p, float v) { *p = v; }
};
template <> struct CacheVec<__nv_bfloat16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void load(const __nv_bfloat16 *p, float *o) {
        const uint4 v = *reinterpret_cast<const uint4 *>(p);
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            o[2 * i] = __uint_as_float(w[i] << 16);
            o[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
        }
    }
    static __device__ __forceinline__ float round(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }
    static __device__ __forceinline__ void store(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }
};

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// One warp: raw head (global) -> dst (shared, `pad` floats, zero-filled past dim): optional RMS norm with a gain, then
// rotation of the pairs (i, i + half), then a factor.
__device__ __forceinline__ void prep_head(const float *src, int dim, int pad, const float *gain, float eps, const skn_rot &rot, int64_t row,
                                          float mul, float *dst) {
    const int lane = threadIdx.x & 31;
    float ss = 0.f;
    for (int d = lane; d < pad; d += 32) {
        const float v = d < dim ? __ldcg(src + d) : 0.f;
        dst[d] = v;
        ss = fmaf(v, v, ss);
    }
    if (gain) {
        const float r = 1.f / sqrtf(warp_sum(ss) / (float)dim + eps);
        for (int d = lane; d < dim; d += 32) dst[d] = dst[d] * r * __ldg(gain + d);
    }
    __syncwarp();
    for (int i = lane; i < rot.half; i += 32) {
        const float2 cs = __ldcg(rot.table + row * rot.ld + i);
        const float u = dst[i], v = dst[i + rot.half];
        dst[i] = u * cs.x - v * cs.y;
        dst[i + rot.half] = v * cs.x + u * cs.y;
    }
    __syncwarp();
    if (mul != 1.f)
        for (int d = lane; d < dim; d += 32) dst[d] *= mul;
    __syncwarp();
}

// first key that the query at position p sees
__device__ __forceinline__ int first_visible(const skn_attn_args &a, int p) {
    return a.chunk > 0 ? p / a.chunk * a.chunk : a.window > 0 ? max(0, p - a.window + 1) : 0;
}

__device__ __forceinline__ void put_out(const skn_rows_out &o, int64_t m, int64_t c, float v) {
    if (o.y32) o.y32[m * o.ld32 + c] = v;
    if (o.y16) o.y16[m * o.ld16 + c] = __float2bfloat16_rn(v);
}

// ---- attention over a split of the keys ---------------------------------------------------------------------------
// smem (floats): q [RT][kp] | key [kp] | value [vp] | weights [RT][KS] | red [partial sums][RT][vp]
template <class CT, int RT>
static size_t attn_split_smem(int kp, int vp) {
    const int ng = vp / CacheVec<CT>::N, parts = ng <= 32 && 32 % ng == 0 ? MIX_THREADS / 32 : MIX_THREADS / ng;
    return ((size_t)RT * kp + kp + vp + RT * KS + (size_t)parts * RT * vp) * sizeof(float);
}

template <class CT, int RT, bool APPEND>
__device__ void attn_split(const skn_attn_args &a, const skn_step &st, const CT *__restrict__ kc_, const CT *__restrict__ vc_, int G, int cap, int dim,
                           int vdim, int kp, int vp, int vld, int split, int max_splits, int hg, int m, float *sm) {
    constexpr int VE = CacheVec<CT>::N;
    __shared__ float s_red[MIX_THREADS / 32][RT], s_max[RT], s_sum[RT];
    __shared__ bool s_last;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int R = a.heads / G, ngr = (R + RT - 1) / RT, g = hg / ngr, sub = hg % ngr;
    const int h0 = g * R + sub * RT, nh = min(RT, R - sub * RT);
    const int seq = m / st.T, slot = st.slot0 + seq;
    const int p = min(st.pos[slot] + m % st.T, st.max_pos - 1);
    const int lo = first_visible(a, p);
    const int live = (p - lo) / KS + 1;
    if (split >= live) return;
    const int j0 = lo + split * KS, nk = min(KS, p + 1 - j0);
    const bool newest = APPEND && split == live - 1;       // this split ends with the step's own key
    float *qs = sm, *kn = qs + RT * kp, *vn = kn + kp, *ws = vn + vp, *red = ws + RT * KS;
    const size_t head_rows = ((size_t)slot * G + g) * cap;
    CT *kc = const_cast<CT *>(kc_) + head_rows * kp, *vc = const_cast<CT *>(vc_) + head_rows * vld;
    // keys and values on their way into L2 while the query is prepared: two threads per key
    const int key = tid >> 1, half = tid & 1;
    const int kslot = (j0 + key) % cap;
    if (key < nk) {
        const char *kr = reinterpret_cast<const char *>(kc + (size_t)kslot * kp), *vr = reinterpret_cast<const char *>(vc + (size_t)kslot * vld);
        for (int i = half * 128; i < (int)(kp * sizeof(CT)); i += 256) asm volatile("prefetch.global.L2 [%0];" ::"l"(kr + i));
        if (vc != kc)
            for (int i = half * 128; i < (int)(vp * sizeof(CT)); i += 256) asm volatile("prefetch.global.L2 [%0];" ::"l"(vr + i));
    }

    for (int i = warp; i < RT + 2; i += MIX_THREADS / 32) {
        if (i < RT) {
            if (i < nh) prep_head(a.q + (int64_t)m * a.ld + (int64_t)(h0 + i) * dim, dim, kp, a.q_gain, a.eps, a.rot, m, a.scale, qs + i * kp);
            else for (int d = lane; d < kp; d += 32) qs[i * kp + d] = 0.f;
        } else if (newest && i == RT) {
            prep_head(a.k + (int64_t)m * a.ld + (int64_t)g * dim, dim, kp, a.k_gain, a.eps, a.rot, m, 1.f, kn);
            for (int d = lane; d < dim; d += 32) {
                if (sub == 0) CacheVec<CT>::store(kc + (size_t)(p % cap) * kp + d, kn[d]);
                kn[d] = CacheVec<CT>::round(kn[d]);
            }
        } else if (newest) {
            for (int d = lane; d < vp; d += 32) {
                const float v = d < vdim ? __ldcg(a.v + (int64_t)m * a.ld + (int64_t)g * vdim + d) : 0.f;
                if (sub == 0 && d < vdim) CacheVec<CT>::store(vc + (size_t)(p % cap) * vld + d, v);
                vn[d] = CacheVec<CT>::round(v);
            }
        }
    }
    __syncthreads();

    // scores: two threads per key, each takes every other vector of the row
    const bool valid = key < nk, own = newest && key == nk - 1;
    float s[RT];
#pragma unroll
    for (int r = 0; r < RT; ++r) s[r] = 0.f;
    if (valid) {
        const CT *kr = kc + (size_t)kslot * kp;
#pragma unroll 4
        for (int u = half; u < kp / VE; u += 2) {
            float kv[VE];
            if (own) {
#pragma unroll
                for (int e = 0; e < VE; ++e) kv[e] = kn[u * VE + e];
            } else CacheVec<CT>::load(kr + u * VE, kv);
#pragma unroll
            for (int r = 0; r < RT; ++r)
#pragma unroll
                for (int e = 0; e < VE; ++e) s[r] = fmaf(qs[r * kp + u * VE + e], kv[e], s[r]);
        }
    }
#pragma unroll
    for (int r = 0; r < RT; ++r) {
        s[r] += __shfl_xor_sync(0xffffffffu, s[r], 1);
        if (a.softcap > 0.f) s[r] = a.softcap * tanhf(s[r] / a.softcap);
        if (!valid) s[r] = -INFINITY;
        const float wm = warp_max(s[r]);
        if (lane == 0) s_red[warp][r] = wm;
    }
    __syncthreads();
    float mx[RT];
#pragma unroll
    for (int r = 0; r < RT; ++r) {
        mx[r] = s_red[0][r];
#pragma unroll
        for (int w = 1; w < MIX_THREADS / 32; ++w) mx[r] = fmaxf(mx[r], s_red[w][r]);
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < RT; ++r) {
        const float e = valid ? expf(s[r] - mx[r]) : 0.f;
        if (half == 0) ws[r * KS + key] = e;
        const float t = warp_sum(half == 0 ? e : 0.f);
        if (lane == 0) s_red[warp][r] = t;
    }
    __syncthreads();
    if (tid < RT) {
        float t = 0.f;
        for (int w = 0; w < MIX_THREADS / 32; ++w) t += s_red[w][tid];
        s_sum[tid] = t;
    }
#pragma unroll
    for (int r = 0; r < RT; ++r)
        if (tid == r) s_max[r] = mx[r];

    // values: a thread owns one vector of columns and every kl-th key
    const int ng = vp / VE, kl = MIX_THREADS / ng, cg_ = tid % ng, kk = tid / ng;
    float acc[RT][VE];
#pragma unroll
    for (int r = 0; r < RT; ++r)
#pragma unroll
        for (int e = 0; e < VE; ++e) acc[r][e] = 0.f;
    if (kk < kl) {
        const int first = j0 % cap;
#pragma unroll 4
        for (int j = kk; j < nk; j += kl) {
            float vv[VE];
            int sl = first + j;
            if (sl >= cap) sl -= cap;              // (a cache holds at least the keys that one query sees)
            if (newest && j == nk - 1) {
#pragma unroll
                for (int e = 0; e < VE; ++e) vv[e] = vn[cg_ * VE + e];
            } else CacheVec<CT>::load(vc + (size_t)sl * vld + cg_ * VE, vv);
#pragma unroll
            for (int r = 0; r < RT; ++r) {
                const float w = ws[r * KS + j];
#pragma unroll
                for (int e = 0; e < VE; ++e) acc[r][e] = fmaf(w, vv[e], acc[r][e]);
            }
        }
    }
    // a column vector's partial sums: first across the lanes of a warp that hold the same columns, then across the warps
    const bool fold = ng <= 32 && 32 % ng == 0;
    if (fold) {
        for (int o = ng; o < 32; o <<= 1)
#pragma unroll
            for (int r = 0; r < RT; ++r)
#pragma unroll
                for (int e = 0; e < VE; ++e) acc[r][e] += __shfl_xor_sync(0xffffffffu, acc[r][e], o);
    }
    const int part = fold ? warp : kk;
    if (kk < kl && (!fold || lane < ng)) {
#pragma unroll
        for (int r = 0; r < RT; ++r)
#pragma unroll
            for (int e = 0; e < VE; ++e) red[((size_t)part * RT + r) * vp + cg_ * VE + e] = acc[r][e];
    }
    __syncthreads();
    const int nk_l = fold ? MIX_THREADS / 32 : min(kl, nk);
    for (int i = tid; i < nh * vdim; i += MIX_THREADS) {
        const int r = i / vdim, c = i % vdim;
        float o = 0.f;
        for (int k2 = 0; k2 < nk_l; ++k2) o += red[((size_t)k2 * RT + r) * vp + c];
        if (live == 1) put_out(a.out, m, (int64_t)(h0 + r) * vdim + c, o / (a.sink ? s_sum[r] + expf(a.sink[h0 + r] - s_max[r]) : s_sum[r]) * a.out_scale);
        else __stcg(a.scratch + (((size_t)m * a.heads + h0 + r) * max_splits + split) * (vdim + 2) + 2 + c, o);
    }
    if (live == 1) return;
    if (tid < nh) {
        float *rec = a.scratch + (((size_t)m * a.heads + h0 + tid) * max_splits + split) * (vdim + 2);
        __stcg(rec, s_max[tid]);
        __stcg(rec + 1, s_sum[tid]);
    }
    __threadfence();
    __syncthreads();
    unsigned *ticket = a.tickets + (size_t)m * a.heads + h0;
    if (tid == 0) s_last = atomicAdd(ticket, 1u) == (unsigned)(live - 1);
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    // weight of every split (in place of the scores): exp(max - top) / sum
    for (int r = warp; r < nh; r += MIX_THREADS / 32) {
        const float *rec = a.scratch + ((size_t)m * a.heads + h0 + r) * max_splits * (vdim + 2);
        float top = -INFINITY;
        for (int x = lane; x < live; x += 32) top = fmaxf(top, __ldcg(rec + (size_t)x * (vdim + 2)));
        top = warp_max(top);
        const float sink = a.sink ? a.sink[h0 + r] : -INFINITY;
        top = fmaxf(top, sink);
        float den = 0.f;
        for (int x = lane; x < live; x += 32) den += expf(__ldcg(rec + (size_t)x * (vdim + 2)) - top) * __ldcg(rec + (size_t)x * (vdim + 2) + 1);
        den = warp_sum(den) + (a.sink ? expf(sink - top) : 0.f);
        for (int x = lane; x < live; x += 32)
            if (x < KS) ws[r * KS + x] = expf(__ldcg(rec + (size_t)x * (vdim + 2)) - top) / den;
        if (lane == 0) { s_max[r] = top; s_sum[r] = den; }
    }
    __syncthreads();
    for (int i = tid; i < nh * vdim; i += MIX_THREADS) {
        const int r = i / vdim, c = i % vdim;
        const float *rec = a.scratch + ((size_t)m * a.heads + h0 + r) * max_splits * (vdim + 2);
        float num = 0.f;
#pragma unroll 8
        for (int x = 0; x < live; ++x) {
            const float f = x < KS ? ws[r * KS + x] : expf(__ldcg(rec + (size_t)x * (vdim + 2)) - s_max[r]) / s_sum[r];
            num = fmaf(f, __ldcg(rec + (size_t)x * (vdim + 2) + 2 + c), num);
        }
        put_out(a.out, m, (int64_t)(h0 + r) * vdim + c, num * a.out_scale);
    }
    if (tid == 0) *ticket = 0;
}

// ---- retention, one token ----------------------------------------------------------------------------------------
// smem (floats): q [dk] | k [dk] | v [vp] | o [vp] | red [MIX_THREADS * 4]
static size_t ret_step_smem(int dk, int vp) { return ((size_t)2 * ((dk + 3) / 4 * 4) + 2 * vp + MIX_THREADS * 4) * sizeof(float); }

__device__ void ret_step(const skn_ret_args &r, const skn_step &st, float *__restrict__ S, int H, int dk, int dv, int vp, int h, int m, float *sm) {
    __shared__ float s_w[MIX_THREADS / 32];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, dkp = (dk + 3) / 4 * 4;
    float *qs = sm, *ks = qs + dkp, *vs = ks + dkp, *os = vs + vp, *red = os + vp;
    const int slot = st.slot0 + m / st.T;
    const bool fresh = st.pos[slot] == 0;
    const float decay = __ldg(r.powers + (size_t)h * (SKN_RET_CHUNK + 1) + 1);
    if (warp == 0) prep_head(r.q + (int64_t)m * r.ld + (int64_t)h * dk, dk, dk, nullptr, 0.f, r.rot, m, 1.f, qs);
    else if (warp == 1) prep_head(r.k + (int64_t)m * r.ld + (int64_t)h * dk, dk, dk, nullptr, 0.f, r.rot, m, r.k_scale, ks);
    else if (warp == 2)
        for (int d = lane; d < vp; d += 32) vs[d] = d < dv ? __ldcg(r.v + (int64_t)m * r.ld + (int64_t)h * dv + d) : 0.f;
    __syncthreads();
    float *base = S + ((size_t)slot * H + h) * dk * vp;
    // the column groups that do not fill the block at once take further turns
    for (int c0 = 0; c0 < vp / 4; c0 += MIX_THREADS) {
        const int nc = min(MIX_THREADS, vp / 4 - c0), lanes = MIX_THREADS / nc, cg_ = tid % nc, rl = tid / nc;
        if (rl < lanes) {
            const int c = (c0 + cg_) * 4;
            const float4 v = *reinterpret_cast<const float4 *>(vs + c);
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
            for (int i = rl; i < dk; i += lanes) {
                float4 *p = reinterpret_cast<float4 *>(base + (size_t)i * vp + c);
                float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *p;
                const float k = ks[i], q = qs[i];
                s.x = fmaf(decay, s.x, k * v.x);
                s.y = fmaf(decay, s.y, k * v.y);
                s.z = fmaf(decay, s.z, k * v.z);
                s.w = fmaf(decay, s.w, k * v.w);
                *p = s;
                o.x = fmaf(q, s.x, o.x);
                o.y = fmaf(q, s.y, o.y);
                o.z = fmaf(q, s.z, o.z);
                o.w = fmaf(q, s.w, o.w);
            }
            *reinterpret_cast<float4 *>(red + ((size_t)rl * nc + cg_) * 4) = o;
        }
        __syncthreads();
        for (int i = tid; i < nc * 4; i += MIX_THREADS) {
            float t = 0.f;
            for (int x = 0; x < min(lanes, dk); ++x) t += red[(size_t)x * nc * 4 + i];
            os[c0 * 4 + i] = t;
        }
        __syncthreads();
    }
    float ss = 0.f;
    for (int d = tid; d < dv; d += MIX_THREADS) ss = fmaf(os[d], os[d], ss);
    ss = warp_sum(ss);
    if (lane == 0) s_w[warp] = ss;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < MIX_THREADS / 32; ++w) t += s_w[w];
    const float rs = 1.f / sqrtf(t / (float)dv + r.eps);
    for (int d = tid; d < dv; d += MIX_THREADS) {
        const float gt = __ldcg(r.g + (int64_t)m * r.ld + (int64_t)h * dv + d);
        put_out(r.out, m, (int64_t)h * dv + d, os[d] * rs * (gt / (1.f + expf(-gt))) * r.out_scale);
    }
}

template <class CT, int RT>
__global__ void __launch_bounds__(MIX_THREADS, 4)
skn_mix_decode_kernel(skn_attn_args a, skn_ret_args r, skn_step st, const CT *kc, const CT *vc, int G, int cap, int dim, int vdim, int kp,
                      int vp, int vld, int max_splits, int n_attn, float *S, int RH, int rdk, int rdv, int rvp) {
    extern __shared__ __align__(16) float sm[];
    // the next launch starts only when this one's CTAs end (no early trigger): the weights it would stream meanwhile make
    // every step of this chain of dependent loads wait longer
    skn_pdl_wait();
    const int m = blockIdx.y, b = blockIdx.x;
    if (b < n_attn) attn_split<CT, RT, true>(a, st, kc, vc, G, cap, dim, vdim, kp, vp, vld, b % max_splits, max_splits, b / max_splits, m, sm);
    else ret_step(r, st, S, RH, rdk, rdv, rvp, b - n_attn, m, sm);
}

template <class CT, int RT>
__global__ void __launch_bounds__(MIX_THREADS)
skn_attn_rows_kernel(skn_attn_args a, skn_step st, const CT *kc, const CT *vc, int G, int cap, int dim, int vdim, int kp, int vp, int vld,
                     int max_splits) {
    extern __shared__ __align__(16) float sm[];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    attn_split<CT, RT, false>(a, st, kc, vc, G, cap, dim, vdim, kp, vp, vld, blockIdx.x % max_splits, max_splits, blockIdx.x / max_splits, blockIdx.y, sm);
}

template <class CT, int RT>
static cudaError_t launch_decode_t(const skn_step &s, const skn_attn_args *a, const skn_ret_args *r, bool rows_only, cudaStream_t st) {
    skn_attn_args aa = {};
    skn_ret_args rr = {};
    int G = 1, cap = 1, dim = 1, vdim = 1, kp = 16, vp = 16, vld = 16, ms = 1, n_attn = 0, RH = 0, dk = 1, dv = 1, rvp = 4;
    const CT *kc = nullptr, *vc = nullptr;
    float *S = nullptr;
    size_t smem = 0;
    if (a) {
        aa = *a;
        G = a->kv->n_kv_heads; cap = a->kv->capacity; dim = a->kv->head_dim; vdim = a->kv->v_dim; kp = a->kv->k_pitch; vp = a->kv->v_pitch;
        vld = a->kv->v_stride;
        kc = (const CT *)a->kv->d_k;
        vc = (const CT *)a->kv->d_v;
        ms = skn_attn_splits(a->chunk > 0 ? a->chunk : a->window, s.max_pos);
        n_attn = ms * G * ((a->heads / G + RT - 1) / RT);
        smem = attn_split_smem<CT, RT>(kp, vp);
    }
    if (r) {
        rr = *r;
        S = r->state->d;
        RH = r->state->heads; dk = r->state->k_dim; dv = r->state->v_dim; rvp = r->state->v_pitch;
        const size_t b = ret_step_smem(dk, rvp);
        if (b > smem) smem = b;
    }
    const dim3 grid(n_attn + (rows_only ? 0 : RH), s.n_seqs * s.T);
    if (rows_only) {
        auto kern = skn_attn_rows_kernel<CT, RT>;
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
        if (e != cudaSuccess) return e;
        return skn_launch_pdl(kern, grid, dim3(MIX_THREADS), smem, st, 1, aa, s, kc, vc, G, cap, dim, vdim, kp, vp, vld, ms);
    }
    auto kern = skn_mix_decode_kernel<CT, RT>;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
    if (e != cudaSuccess) return e;
    return skn_launch_pdl(kern, grid, dim3(MIX_THREADS), smem, st, 1, aa, rr, s, kc, vc, G, cap, dim, vdim, kp, vp, vld, ms, n_attn, S, RH, dk, dv, rvp);
}

static cudaError_t launch_split(const skn_step &s, const skn_attn_args *a, const skn_ret_args *r, bool rows_only, cudaStream_t st) {
    const int R = a ? a->heads / a->kv->n_kv_heads : 1;
    if (a && a->kv->dtype == SKN_KV_BF16)
        return R > 2 ? launch_decode_t<__nv_bfloat16, 4>(s, a, r, rows_only, st) : R == 2 ? launch_decode_t<__nv_bfloat16, 2>(s, a, r, rows_only, st)
                                                                                : launch_decode_t<__nv_bfloat16, 1>(s, a, r, rows_only, st);
    return R > 2 ? launch_decode_t<float, 4>(s, a, r, rows_only, st) : R == 2 ? launch_decode_t<float, 2>(s, a, r, rows_only, st)
                                                                   : launch_decode_t<float, 1>(s, a, r, rows_only, st);
}

cudaError_t skn_launch_attn_rows(const skn_step &s, const skn_attn_args &a, cudaStream_t st) { return launch_split(s, &a, nullptr, true, st); }

cudaError_t skn_launch_mix_decode(skn_ctx *, const skn_step &s, const skn_attn_args *a, const skn_ret_args *r, cudaStream_t st) {
    if (s.T != 1) return cudaErrorInvalidValue;
    return launch_split(s, a, r, false, st);
}

// ---- many tokens: heads prepared, keys and values into the cache --------------------------------------------------
struct prep_args {
    int H, G, dim, vdim, kp, vp, cap;
    int RH, rdk;
};

template <class CT>
__global__ void __launch_bounds__(256)
skn_head_prep_kernel(skn_attn_args a, skn_ret_args r, skn_step st, prep_args p, CT *kc, CT *vc) {
    extern __shared__ __align__(16) float sm[];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, m = blockIdx.x;
    const int width = max(p.kp, p.rdk);
    float *buf = sm + (size_t)warp * width;
    const int slot = st.slot0 + m / st.T, pos = min(st.pos[slot] + m % st.T, st.max_pos - 1);
    const int nq = a.q16 ? p.H : 0, units = nq + 2 * p.G + 2 * p.RH;
    for (int u = warp; u < units; u += 8) {
        if (u < nq) {
            prep_head(a.q + (int64_t)m * a.ld + (int64_t)u * p.dim, p.dim, p.kp, a.q_gain, a.eps, a.rot, m, 1.f, buf);
            for (int d = lane; d < p.kp; d += 32) a.q16[((int64_t)m * p.H + u) * p.kp + d] = __float2bfloat16_rn(buf[d]);
        } else if (u < nq + p.G) {
            const int g = u - nq;
            prep_head(a.k + (int64_t)m * a.ld + (int64_t)g * p.dim, p.dim, p.kp, a.k_gain, a.eps, a.rot, m, 1.f, buf);
            CT *dst = kc + (((size_t)slot * p.G + g) * p.cap + pos % p.cap) * p.kp;
            for (int d = lane; d < p.dim; d += 32) CacheVec<CT>::store(dst + d, buf[d]);
        } else if (u < nq + 2 * p.G) {
            const int g = u - nq - p.G;
            CT *dst = vc + (((size_t)slot * p.G + g) * p.cap + pos % p.cap) * p.vp;
            for (int d = lane; d < p.vdim; d += 32) CacheVec<CT>::store(dst + d, __ldcg(a.v + (int64_t)m * a.ld + (int64_t)g * p.vdim + d));
        } else {
            const int i = u - nq - 2 * p.G, h = i >> 1;
            float *src = ((i & 1) ? r.k : r.q) + (int64_t)m * r.ld + (int64_t)h * p.rdk;
            prep_head(src, p.rdk, p.rdk, nullptr, 0.f, r.rot, m, (i & 1) ? r.k_scale : 1.f, buf);
            for (int d = lane; d < p.rdk; d += 32) src[d] = buf[d];
        }
        __syncwarp();
    }
}

// ---- attention on the tensor cores ---------------------------------------------------------------------------------
constexpr int ATQ = 64, ATK = 32;      // queries and keys of a tile
constexpr int AT_THREADS = ATQ * 2;    // a warp owns 16 queries

// tanh through one exponential; absolute error a few 1e-7
__device__ __forceinline__ float tanh_exp(float y) {
    const float t = __expf(2.f * fminf(fmaxf(y, -20.f), 20.f));
    return 1.f - __fdividef(2.f, t + 1.f);
}

template <int DV>
__global__ void __launch_bounds__(AT_THREADS, DV <= 128 ? 3 : 1)
skn_attn_tc_kernel(skn_attn_args a, skn_step st, skn_attn_keys src) {
    extern __shared__ __align__(16) uint8_t smb[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kp = src.kp, vp = src.vp, cap = src.cap, vdim = src.vdim;
    const int ks = kp + 8, vs = DV + 8;                                  // row strides in elements
    __nv_bfloat16 *Q = reinterpret_cast<__nv_bfloat16 *>(smb), *K = Q + ATQ * ks, *V = K + 2 * ATK * ks;
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int t0 = (gridDim.x - 1 - blockIdx.x) * ATQ, h = blockIdx.y, seq = blockIdx.z, slot = st.slot0 + seq, g = h / src.group;
    const int p0 = st.pos[slot], nq = min(ATQ, st.T - t0);
    const int pf = p0 + t0, pl = pf + nq - 1;                            // first and last query position
    const int lo = first_visible(a, pf);
    const int tiles = (pl - lo) / ATK + 1;
    const __nv_bfloat16 *kc = src.k + slot * src.k_slot + g * src.k_head, *vc = src.v + slot * src.v_slot + g * src.v_head;
    const __nv_bfloat16 *kc2 = src.k2 ? src.k2 + slot * src.k2_slot : nullptr;

    const int slot0 = lo % cap;
    const bool idle = warp * 16 >= nq;                                   // none of this warp's queries exist
    // four threads per key row (two per query row), every fourth 16-byte piece each
    const int cr = tid >> 2, cc = tid & 3;
    auto load_tile = [&](int t, int buf) {
        const int j = lo + t * ATK + cr;
        const bool in = j <= pl;
        int sl = slot0 + t * ATK + cr;
        if (sl >= cap) sl %= cap;
        const __nv_bfloat16 *kr = kc + sl * src.k_row, *vr = vc + sl * src.v_row, *kr2 = kc2 + sl * src.k2_row - src.k1;
        const uint32_t kd = skn_smem_u32(K + ((size_t)buf * ATK + cr) * ks), vd = skn_smem_u32(V + ((size_t)buf * ATK + cr) * vs);
        for (int c = cc * 8; c < kp; c += 32) cp_async16(kd + c * 2, (c < src.k1 ? kr : kr2) + c, in);
#pragma unroll
        for (int c = cc * 8; c < DV; c += 32) cp_async16(vd + c * 2, vr + (c < vp ? c : 0), in && c < vp);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    {
        const int r = tid >> 1;
        const __nv_bfloat16 *q = a.q16 + (((int64_t)seq * st.T + t0 + (r < nq ? r : 0)) * a.heads + h) * kp;
        for (int c = (tid & 1) * 8; c < kp; c += 16) cp_async16(skn_smem_u32(Q + (size_t)r * ks + c), q + c, r < nq);
    }
    load_tile(0, 0);

    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    // a sink is one more key without a value: it opens the running maximum and, once per row, the sum
    const float L2E = 1.4426950408889634f, sink = a.sink ? a.sink[h] * L2E : -INFINITY, l0 = a.sink && (lane & 3) == 0 ? 1.f : 0.f;
    float mrow[2] = {sink, sink}, lrow[2] = {l0, l0};
    const int r0 = warp * 16 + (lane >> 2);
    const int qi[2] = {pf + r0, pf + r0 + 8};
    int qlo[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) qlo[i] = first_visible(a, qi[i]);
    const int w0 = pf + warp * 16, wlo = first_visible(a, w0), whi = first_visible(a, w0 + 15);
    const float inv_cap = a.softcap > 0.f ? a.scale / a.softcap : 0.f;

    for (int t = 0; t < tiles; ++t) {
        const int buf = t & 1;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (t + 1 < tiles) load_tile(t + 1, buf ^ 1);
        const int j0 = lo + t * ATK;
        // tiles that none of the warp's queries sees: past its last query, or in an earlier chunk than its first
        if (idle || j0 > w0 + 15 || j0 + ATK <= wlo) {
            __syncthreads();
            continue;
        }
        const bool masked = j0 + ATK - 1 > w0 || j0 < whi;               // some pair of this tile is invisible
        float s[ATK / 8][4];
#pragma unroll
        for (int i = 0; i < ATK / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
        const __nv_bfloat16 *Kb = K + (size_t)buf * ATK * ks, *Vb = V + (size_t)buf * ATK * vs;
        for (int kk = 0; kk < kp; kk += 16) {
            uint32_t af[4];
            ldsm4(af, skn_smem_u32(Q + (size_t)(warp * 16 + (lane & 15)) * ks + kk + (lane >> 4) * 8));
#pragma unroll
            for (int n = 0; n < ATK / 16; ++n) {
                uint32_t bf[4];
                ldsm4(bf, skn_smem_u32(Kb + (size_t)(n * 16 + (lane & 7) + ((lane >> 4) << 3)) * ks + kk + ((lane >> 3) & 1) * 8));
                mma_bf16(s[2 * n], af, bf[0], bf[1]);
                mma_bf16(s[2 * n + 1], af, bf[2], bf[3]);
            }
        }
        float mx[2] = {mrow[0], mrow[1]};
#pragma unroll
        for (int n = 0; n < ATK / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = e >> 1, j = j0 + n * 8 + (lane & 3) * 2 + (e & 1);
                float v = a.softcap > 0.f ? a.softcap * tanh_exp(s[n][e] * inv_cap) : s[n][e] * a.scale;
                v = !masked || (j <= qi[i] && j >= qlo[i]) ? v * L2E : -INFINITY;
                s[n][e] = v;
                mx[i] = fmaxf(mx[i], v);
            }
        float corr[2], base[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
            base[i] = mx[i] == -INFINITY ? 0.f : mx[i];
            corr[i] = exp2f(mrow[i] - base[i]);
            mrow[i] = mx[i];
            lrow[i] *= corr[i];
        }
#pragma unroll
        for (int n = 0; n < ATK / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                s[n][e] = exp2f(s[n][e] - base[e >> 1]);
                lrow[e >> 1] += s[n][e];
            }
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) {
            o[i][0] *= corr[0]; o[i][1] *= corr[0];
            o[i][2] *= corr[1]; o[i][3] *= corr[1];
        }
#pragma unroll
        for (int kk = 0; kk < ATK / 16; ++kk) {
            uint32_t hi[4], lw[4];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float *w = s[2 * kk + (x >> 1)];
                const float w0 = w[(x & 1) * 2], w1 = w[(x & 1) * 2 + 1];
                hi[x] = pack_bf16(w0, w1);
                lw[x] = pack_bf16(w0 - __uint_as_float(hi[x] << 16), w1 - __uint_as_float(hi[x] & 0xFFFF0000u));
            }
#pragma unroll
            for (int n = 0; n < DV / 16; ++n) {
                uint32_t bf[4];
                ldsm4t(bf, skn_smem_u32(Vb + (size_t)(kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + n * 16 + (lane >> 4) * 8));
                mma_bf16(o[2 * n], hi, bf[0], bf[1]);
                mma_bf16(o[2 * n + 1], hi, bf[2], bf[3]);
                mma_bf16(o[2 * n], lw, bf[0], bf[1]);
                mma_bf16(o[2 * n + 1], lw, bf[2], bf[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        lrow[i] += __shfl_xor_sync(0xffffffffu, lrow[i], 1);
        lrow[i] += __shfl_xor_sync(0xffffffffu, lrow[i], 2);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = r0 + i * 8;
        if (r >= nq) continue;
        const float f = a.out_scale / lrow[i];
        const int64_t m = (int64_t)seq * st.T + t0 + r;
#pragma unroll
        for (int n = 0; n < DV / 8; ++n) {
            const int c = n * 8 + (lane & 3) * 2;
#pragma unroll
            for (int e = 0; e < 2; ++e)
                if (c + e < vdim) {
                    float v = o[n][i * 2 + e] * f;
                    if (a.gate) v *= __fdividef(1.f, 1.f + __expf(fminf(-__ldcg(a.gate + m * a.ld_gate + (int64_t)h * vdim + c + e), 80.f)));
                    put_out(a.out, m, (int64_t)h * vdim + c + e, v);
                }
        }
    }
}

template <int DV>
static cudaError_t launch_attn_tc(const skn_step &s, const skn_attn_args &a, const skn_attn_keys &k, cudaStream_t st) {
    auto kern = skn_attn_tc_kernel<DV>;
    const size_t smem = ((size_t)(ATQ + 2 * ATK) * (k.kp + 8) + (size_t)2 * ATK * (DV + 8)) * 2;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return e;
    return skn_launch_pdl(kern, dim3((s.T + ATQ - 1) / ATQ, a.heads, s.n_seqs), dim3(AT_THREADS), smem, st, 1, a, s, k);
}

cudaError_t skn_launch_attn_tiles(const skn_step &s, const skn_attn_args &a, const skn_attn_keys &k, cudaStream_t st) {
    const int vp = k.vp;
    return vp <= 32 ? launch_attn_tc<32>(s, a, k, st) : vp <= 64 ? launch_attn_tc<64>(s, a, k, st) : vp <= 96 ? launch_attn_tc<96>(s, a, k, st)
           : vp <= 128 ? launch_attn_tc<128>(s, a, k, st) : vp <= 192 ? launch_attn_tc<192>(s, a, k, st) : launch_attn_tc<256>(s, a, k, st);
}

static skn_attn_keys cache_keys(const skn_kvcache *kv, int heads) {
    skn_attn_keys k = {};
    k.kp = k.k1 = kv->k_pitch; k.vp = kv->v_pitch; k.vdim = kv->v_dim; k.cap = kv->capacity; k.group = heads / kv->n_kv_heads;
    k.k = (const __nv_bfloat16 *)kv->d_k; k.k_row = kv->k_pitch; k.k_head = (int64_t)kv->capacity * kv->k_pitch; k.k_slot = k.k_head * kv->n_kv_heads;
    k.v = (const __nv_bfloat16 *)kv->d_v; k.v_row = kv->v_stride; k.v_head = (int64_t)kv->capacity * kv->v_stride; k.v_slot = k.v_head * kv->n_kv_heads;
    return k;
}

bool skn_attn_tiles_fit(int kp, int vp) { return kp <= 256 && vp <= 256; }
bool skn_chunk_attn_tc(const skn_kvcache *kv) { return kv->dtype == SKN_KV_BF16 && skn_attn_tiles_fit(kv->k_pitch, kv->v_pitch); }

// ---- retention in chunks --------------------------------------------------------------------------------------------
constexpr int RC = SKN_RET_CHUNK;

// what chunk c adds to the state by its end: sum over its tokens j of decay^(L - 1 - j) k_j v_j^T.  CTA: a 64 x 64 tile.
__global__ void __launch_bounds__(256)
skn_ret_chunk_kernel(skn_ret_args r, int T, int H, int dk, int dv, int vp, int nchunks, int vtiles) {
    __shared__ __align__(16) float kt[RC][64], vt[RC][64];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int c = blockIdx.x, h = blockIdx.y % H, seq = blockIdx.y / H, i0 = (blockIdx.z / vtiles) * 64, j0 = (blockIdx.z % vtiles) * 64;
    const int t0 = c * RC, L = min(RC, T - t0);
    const float *pw = r.powers + (size_t)h * (RC + 1);
    const int64_t row0 = (int64_t)seq * T + t0;
    for (int i = threadIdx.x; i < RC * 64; i += 256) {
        const int t = i >> 6, d = i & 63;
        kt[t][d] = t < L && i0 + d < dk ? __ldcg(r.k + (row0 + t) * r.ld + (int64_t)h * dk + i0 + d) * pw[L - 1 - t] : 0.f;
        vt[t][d] = t < L && j0 + d < dv ? __ldcg(r.v + (row0 + t) * r.ld + (int64_t)h * dv + j0 + d) : 0.f;
    }
    __syncthreads();
    const int ti = (threadIdx.x >> 4) * 4, tj = (threadIdx.x & 15) * 4;
    float acc[4][4] = {};
    for (int t = 0; t < L; ++t) {
        const float4 a = *reinterpret_cast<const float4 *>(&kt[t][ti]), b = *reinterpret_cast<const float4 *>(&vt[t][tj]);
        const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    float *out = r.chunks + ((((size_t)seq * nchunks + c) * H + h) * dk) * vp;
#pragma unroll
    for (int i = 0; i < 4; ++i)
        if (i0 + ti + i < dk && j0 + tj < vp)
            *reinterpret_cast<float4 *>(out + (size_t)(i0 + ti + i) * vp + j0 + tj) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
}

// chunk sums -> states at the chunk starts (in place), and the state after the step
__global__ void __launch_bounds__(128)
skn_ret_scan_kernel(skn_ret_args r, skn_step st, float *S, int H, int dk, int vp, int nchunks) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int seq = blockIdx.y, slot = st.slot0 + seq, T = st.T;
    const int64_t per = (int64_t)H * dk * (vp / 4), i = (int64_t)blockIdx.x * 128 + threadIdx.x;
    if (i >= per) return;
    const int h = (int)(i / ((int64_t)dk * (vp / 4)));
    const float *pw = r.powers + (size_t)h * (RC + 1);
    float4 *p = reinterpret_cast<float4 *>(r.chunks) + (size_t)seq * nchunks * per + i;
    float4 *sp = reinterpret_cast<float4 *>(S) + (size_t)slot * per + i;
    float4 s = st.pos[slot] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *sp;
    const float full = pw[RC], tail = pw[T - (nchunks - 1) * RC];
    for (int c0 = 0; c0 < nchunks; c0 += 8) {
        float4 a[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (c0 + u < nchunks) a[u] = __ldcg(p + (size_t)(c0 + u) * per);
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (c0 + u < nchunks) {
                __stcg(p + (size_t)(c0 + u) * per, s);
                const float d = c0 + u == nchunks - 1 ? tail : full;
                s = make_float4(fmaf(d, s.x, a[u].x), fmaf(d, s.y, a[u].y), fmaf(d, s.z, a[u].z), fmaf(d, s.w, a[u].w));
            }
    }
    *sp = s;
}

// rows of O (shared): divided by their root mean square, gated, scaled, stored
__device__ __forceinline__ void ret_finish(const skn_ret_args &r, const float *O, int os, int64_t row0, int L, int h, int dv) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int t = warp; t < L; t += 8) {
        float ss = 0.f;
        for (int d = lane; d < dv; d += 32) ss = fmaf(O[t * os + d], O[t * os + d], ss);
        const float rs = r.out_scale / sqrtf(warp_sum(ss) / (float)dv + r.eps);
        for (int d = lane; d < dv; d += 32) {
            const float g = __ldcg(r.g + (row0 + t) * r.ld + (int64_t)h * dv + d);
            put_out(r.out, row0 + t, (int64_t)h * dv + d, O[t * os + d] * rs * (g / (1.f + expf(-g))));
        }
    }
}

// outputs of one chunk: o_i = sum_{j <= i} decay^(i - j) (q_i . k_j) v_j + decay^(i + 1) S^T q_i, then normalised and gated.
// smem (floats): A [RC][RC + 4] | x [32][RC + 4] | y [32][68] | o [RC][vw + 4], vw = dv rounded up to 64
static size_t ret_out_smem(int dv) { return ((size_t)RC * (RC + 4) + 32 * (RC + 4) + 32 * 68 + (size_t)RC * ((dv + 63) / 64 * 64 + 4)) * sizeof(float); }

__global__ void __launch_bounds__(256)
skn_ret_out_kernel(skn_ret_args r, int T, int H, int dk, int dv, int vp, int nchunks) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float pw[RC + 1];
    constexpr int AS = RC + 4;
    const int vw = (dv + 63) / 64 * 64, os = vw + 4;
    float *A = sm, *X = A + RC * AS, *Y = X + 32 * AS, *O = Y + 32 * 68;
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int tid = threadIdx.x, c = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, t0 = c * RC, L = min(RC, T - t0);
    const int64_t row0 = (int64_t)seq * T + t0;
    const float *q = r.q + row0 * r.ld + (int64_t)h * dk, *k = r.k + row0 * r.ld + (int64_t)h * dk, *v = r.v + row0 * r.ld + (int64_t)h * dv;
    if (tid <= RC) pw[tid] = r.powers[(size_t)h * (RC + 1) + tid];
    const int ti = (tid >> 4) * 4, tj = (tid & 15) * 4;
    float acc[4][4] = {};
    for (int d0 = 0; d0 < dk; d0 += 32) {
        __syncthreads();
        for (int i = tid; i < RC * 32; i += 256) {
            const int t = i >> 5, d = i & 31;
            const bool in = t < L && d0 + d < dk;
            X[d * AS + t] = in ? __ldcg(q + (int64_t)t * r.ld + d0 + d) : 0.f;
            Y[d * 68 + t] = in ? __ldcg(k + (int64_t)t * r.ld + d0 + d) : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int d = 0; d < 32; ++d) {
            const float4 a = *reinterpret_cast<const float4 *>(X + d * AS + ti), b = *reinterpret_cast<const float4 *>(Y + d * 68 + tj);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
    }
    // stored transposed: A[j][i]
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) A[(tj + j) * AS + ti + i] = tj + j <= ti + i ? acc[i][j] * pw[ti + i - tj - j] : 0.f;
    const float *S = r.chunks + ((((size_t)seq * nchunks + c) * H + h) * dk) * vp;
    for (int v0 = 0; v0 < vw; v0 += 64) {
        float o[4][4] = {};
        for (int j0 = 0; j0 < RC; j0 += 32) {
            __syncthreads();
            for (int i = tid; i < 32 * 64; i += 256) {
                const int j = i >> 6, d = i & 63;
                Y[j * 68 + d] = j0 + j < L && v0 + d < dv ? __ldcg(v + (int64_t)(j0 + j) * r.ld + v0 + d) : 0.f;
            }
            __syncthreads();
#pragma unroll 8
            for (int j = 0; j < 32; ++j) {
                const float4 a = *reinterpret_cast<const float4 *>(A + (j0 + j) * AS + ti), b = *reinterpret_cast<const float4 *>(Y + j * 68 + tj);
                const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
                for (int x = 0; x < 4; ++x)
#pragma unroll
                    for (int y = 0; y < 4; ++y) o[x][y] = fmaf(av[x], bv[y], o[x][y]);
            }
        }
        float p[4][4] = {};
        for (int d0 = 0; d0 < dk; d0 += 32) {
            __syncthreads();
            for (int i = tid; i < RC * 32; i += 256) {
                const int t = i >> 5, d = i & 31;
                X[d * AS + t] = t < L && d0 + d < dk ? __ldcg(q + (int64_t)t * r.ld + d0 + d) : 0.f;
            }
            for (int i = tid; i < 32 * 64; i += 256) {
                const int d = i >> 6, x = i & 63;
                Y[d * 68 + x] = d0 + d < dk && v0 + x < vp ? __ldcg(S + (size_t)(d0 + d) * vp + v0 + x) : 0.f;
            }
            __syncthreads();
#pragma unroll 8
            for (int d = 0; d < 32; ++d) {
                const float4 a = *reinterpret_cast<const float4 *>(X + d * AS + ti), b = *reinterpret_cast<const float4 *>(Y + d * 68 + tj);
                const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
                for (int x = 0; x < 4; ++x)
#pragma unroll
                    for (int y = 0; y < 4; ++y) p[x][y] = fmaf(av[x], bv[y], p[x][y]);
            }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int y = 0; y < 4; ++y) O[(ti + x) * os + v0 + tj + y] = fmaf(pw[ti + x + 1], p[x][y], o[x][y]);
    }
    __syncthreads();
    ret_finish(r, O, os, row0, L, h, dv);
}

// ---- retention chunks on the tensor cores -----------------------------------------------------------------------------
// Every fp32 operand enters as the sum of two tf32 terms and three products are formed (the lowest is below fp32
// rounding), summed in fp32: the results carry fp32 accuracy.  Fragments are read from fp32 rows in shared memory; row
// strides are 4 (rows along M or N) or 8 (rows along K) banks off a multiple of 32, which keeps the reads conflict-free.
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct TwoTerm { uint32_t hi, lo; };
__device__ __forceinline__ TwoTerm two_term(float x) {
    TwoTerm t;
    t.hi = __float_as_uint(x) & 0xFFFFE000u;
    t.lo = __float_as_uint(x - __uint_as_float(t.hi)) & 0xFFFFE000u;
    return t;
}
// c[n] += A (16 x 8 at rows m, column step k) times B (8 x 8 NT): at(row, k) and bt(k, col) read shared memory
template <int NT, class AT, class BT>
__device__ __forceinline__ void mma_two_term(float (&c)[NT][4], int k, AT at, BT bt) {
    const int g = (threadIdx.x & 31) >> 2, t = threadIdx.x & 3;
    uint32_t ah[4], al[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const TwoTerm x = two_term(at(g + (i & 1) * 8, k + t + (i >> 1) * 4));
        ah[i] = x.hi;
        al[i] = x.lo;
    }
#pragma unroll
    for (int n = 0; n < NT; ++n) {
        const TwoTerm b0 = two_term(bt(k + t, n * 8 + g)), b1 = two_term(bt(k + t + 4, n * 8 + g));
        mma_tf32(c[n], al, b0.hi, b1.hi);
        mma_tf32(c[n], ah, b0.lo, b1.lo);
        mma_tf32(c[n], ah, b0.hi, b1.hi);
    }
}

constexpr int RT2 = 128;              // columns of a tile
constexpr int RKS = RT2 + 8;          // row stride of operands whose rows run along K

// the chunk sums of skn_ret_chunk_kernel, in 128 x 128 tiles; a warp owns 16 rows
__global__ void __launch_bounds__(256)
skn_ret_chunk_tc_kernel(skn_ret_args r, int T, int H, int dk, int dv, int vp, int nchunks, int vtiles) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float pw[RC + 1];
    float *Ks = sm, *Vs = sm + RC * RKS;
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int c = blockIdx.x, h = blockIdx.y % H, seq = blockIdx.y / H, i0 = (blockIdx.z / vtiles) * RT2, j0 = (blockIdx.z % vtiles) * RT2;
    const int t0 = c * RC, L = min(RC, T - t0), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int64_t row0 = (int64_t)seq * T + t0;
    const float *k = r.k + row0 * r.ld + (int64_t)h * dk + i0, *v = r.v + row0 * r.ld + (int64_t)h * dv + j0;
    if (tid <= RC) pw[tid] = r.powers[(size_t)h * (RC + 1) + tid];
    __syncthreads();
#pragma unroll 8
    for (int i = tid; i < RC * RT2; i += 256) {
        const int t = i / RT2, d = i % RT2;
        Ks[t * RKS + d] = t < L && i0 + d < dk ? __ldcg(k + (int64_t)t * r.ld + d) * pw[L - 1 - t] : 0.f;
        Vs[t * RKS + d] = t < L && j0 + d < dv ? __ldcg(v + (int64_t)t * r.ld + d) : 0.f;
    }
    __syncthreads();
    float acc[RT2 / 8][4] = {};
    if (i0 + warp * 16 < dk)
        for (int kk = 0; kk < RC; kk += 8)
            mma_two_term(acc, kk, [&](int m, int x) { return Ks[x * RKS + warp * 16 + m]; }, [&](int x, int n) { return Vs[x * RKS + n]; });
    float *out = r.chunks + ((((size_t)seq * nchunks + c) * H + h) * dk) * vp;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int row = i0 + warp * 16 + (lane >> 2) + e * 8;
        if (row >= dk) continue;
#pragma unroll
        for (int n = 0; n < RT2 / 8; ++n) {
            const int col = j0 + n * 8 + (lane & 3) * 2;
            if (col < vp) *reinterpret_cast<float2 *>(out + (size_t)row * vp + col) = make_float2(acc[n][2 * e], acc[n][2 * e + 1]);
        }
    }
}

// the chunk outputs of skn_ret_out_kernel; warp w owns tokens 16 (w & 3) .. and one half of the columns
// smem (floats): q [RC][dkp + 4] | A [RC][RC + 4] | max(k [RC][dkp + 4], b [32][RKS] and o [RC][vw + 4])
static size_t ret_out_tc_smem(int dk, int dv) {
    const size_t qk = (size_t)RC * ((dk + 31) / 32 * 32 + 4), bo = 32 * RKS + (size_t)RC * ((dv + RT2 - 1) / RT2 * RT2 + 4);
    return (qk + RC * (RC + 4) + (qk > bo ? qk : bo)) * sizeof(float);
}

__global__ void __launch_bounds__(256, 2)
skn_ret_out_tc_kernel(skn_ret_args r, int T, int H, int dk, int dv, int vp, int nchunks) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float pw[RC + 1];
    const int dkp = (dk + 31) / 32 * 32, qs = dkp + 4, vw = (dv + RT2 - 1) / RT2 * RT2, os = vw + 4;
    constexpr int AS = RC + 4;
    float *Q = sm, *A = Q + RC * qs, *Kb = A + RC * AS, *B = Kb, *O = Kb + 32 * RKS;
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, t0 = c * RC, L = min(RC, T - t0);
    const int64_t row0 = (int64_t)seq * T + t0;
    const float *q = r.q + row0 * r.ld + (int64_t)h * dk, *k = r.k + row0 * r.ld + (int64_t)h * dk, *v = r.v + row0 * r.ld + (int64_t)h * dv;
    if (tid <= RC) pw[tid] = r.powers[(size_t)h * (RC + 1) + tid];
    for (int d0 = 0; d0 < dkp; d0 += 32)
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int t = warp + i * 8, d = d0 + lane;
            const bool in = t < L && d < dk;
            Q[t * qs + d] = in ? __ldcg(q + (int64_t)t * r.ld + d) : 0.f;
            Kb[t * qs + d] = in ? __ldcg(k + (int64_t)t * r.ld + d) : 0.f;
        }
    __syncthreads();
    const int m0 = (warp & 3) * 16, half = warp >> 2, g = lane >> 2, t = lane & 3;
    {
        float acc[RC / 16][4] = {};
        const int n0 = half * (RC / 2);
        if (n0 <= m0 + 15)                         // else every pair of this tile lies in the future
            for (int kk = 0; kk < dkp; kk += 8)
                mma_two_term(acc, kk, [&](int m, int x) { return Q[(m0 + m) * qs + x]; }, [&](int x, int n) { return Kb[(n0 + n) * qs + x]; });
#pragma unroll
        for (int n = 0; n < RC / 16; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = m0 + g + (e >> 1) * 8, j = n0 + n * 8 + t * 2 + (e & 1);
                A[i * AS + j] = j <= i ? acc[n][e] * pw[i - j] : 0.f;
            }
    }
    const float *S = r.chunks + ((((size_t)seq * nchunks + c) * H + h) * dk) * vp;
    constexpr int NT = RT2 / 16;
    for (int v0 = 0; v0 < vw; v0 += RT2) {
        float o[NT][4] = {};
        const int c0 = half * (RT2 / 2);
        // tiles of 32 rows: the state's first, then the chunk's values
        const int stiles = dkp / 32, tiles = stiles + (L + 31) / 32;
        float pre[16];
        auto fetch = [&](int x) {
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                const int row = (x < stiles ? x : x - stiles) * 32 + (tid >> 7) + i * 2, col = v0 + (tid & 127);
                if (x < stiles) pre[i] = row < dk && col < vp ? __ldcg(S + (size_t)row * vp + col) : 0.f;
                else pre[i] = row < L && col < dv ? __ldcg(v + (int64_t)row * r.ld + col) : 0.f;
            }
        };
        fetch(0);
        for (int x = 0; x < tiles; ++x) {
            __syncthreads();                       // the tile before (or k) is done with
#pragma unroll
            for (int i = 0; i < 16; ++i) B[((tid >> 7) + i * 2) * RKS + (tid & 127)] = pre[i];
            __syncthreads();
            if (x + 1 < tiles) fetch(x + 1);
            if (x == stiles)
#pragma unroll
                for (int n = 0; n < NT; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) o[n][e] *= pw[m0 + g + (e >> 1) * 8 + 1];
            const float *a = x < stiles ? Q + x * 32 : A + (x - stiles) * 32;
            const int lda = x < stiles ? qs : AS;
            if (x < stiles || (x - stiles) * 32 <= m0 + 15)
#pragma unroll
                for (int kk = 0; kk < 32; kk += 8)
                    mma_two_term(o, kk, [&](int m, int y) { return a[(m0 + m) * lda + y]; }, [&](int y, int n) { return B[y * RKS + c0 + n]; });
        }
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e)
                *reinterpret_cast<float2 *>(O + (m0 + g + e * 8) * os + v0 + c0 + n * 8 + t * 2) = make_float2(o[n][2 * e], o[n][2 * e + 1]);
    }
    __syncthreads();
    ret_finish(r, O, os, row0, L, h, dv);
}

template <class CT>
static cudaError_t launch_prep(const skn_step &s, const skn_attn_args *a, const skn_ret_args *r, cudaStream_t st) {
    prep_args p = {};
    skn_attn_args aa = {};
    skn_ret_args rr = {};
    CT *kc = nullptr, *vc = nullptr;
    p.kp = p.vp = 16; p.cap = 1; p.dim = p.vdim = p.rdk = 1;
    if (a) {
        aa = *a;
        p.H = a->heads; p.G = a->kv->n_kv_heads; p.dim = a->kv->head_dim; p.vdim = a->kv->v_dim; p.kp = a->kv->k_pitch; p.vp = a->kv->v_pitch;
        p.cap = a->kv->capacity;
        kc = (CT *)a->kv->d_k;
        vc = (CT *)a->kv->d_v;
        if (!skn_chunk_attn_tc(a->kv)) aa.q16 = nullptr;
    }
    if (r) {
        rr = *r;
        p.RH = r->state->heads; p.rdk = r->state->k_dim;
    }
    const size_t smem = (size_t)8 * (p.kp > p.rdk ? p.kp : p.rdk) * sizeof(float);
    return skn_launch_pdl(skn_head_prep_kernel<CT>, dim3(s.n_seqs * s.T), dim3(256), smem, st, 1, aa, rr, s, p, kc, vc);
}

cudaError_t skn_launch_mix_prefill(skn_ctx *, const skn_step &s, const skn_attn_args *a, const skn_ret_args *r, cudaStream_t st) {
    cudaError_t e = a && a->kv->dtype == SKN_KV_BF16 ? launch_prep<__nv_bfloat16>(s, a, r, st) : launch_prep<float>(s, a, r, st);
    if (e != cudaSuccess) return e;
    if (a) {
        if (skn_chunk_attn_tc(a->kv)) {
            e = skn_launch_attn_tiles(s, *a, cache_keys(a->kv, a->heads), st);
        } else {
            e = launch_split(s, a, nullptr, true, st);
        }
        if (e != cudaSuccess) return e;
    }
    if (r) {
        const int H = r->state->heads, dk = r->state->k_dim, dv = r->state->v_dim, vp = r->state->v_pitch;
        const int nchunks = (s.T + RC - 1) / RC;
        const bool tc = !r->exact && ret_out_tc_smem(dk, dv) <= 200 * 1024;
        const int tile = tc ? RT2 : 64, kt = (dk + tile - 1) / tile, vt = (dv + tile - 1) / tile;
        const dim3 cgrid(nchunks, H * s.n_seqs, kt * vt), ogrid(nchunks, H, s.n_seqs);
        if (tc) {
            e = cudaFuncSetAttribute(skn_ret_chunk_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 2 * RC * RKS * 4);
            if (e != cudaSuccess) return e;
            e = skn_launch_pdl(skn_ret_chunk_tc_kernel, cgrid, dim3(256), (size_t)2 * RC * RKS * 4, st, 1, *r, s.T, H, dk, dv, vp, nchunks, vt);
        } else {
            e = skn_launch_pdl(skn_ret_chunk_kernel, cgrid, dim3(256), 0, st, 1, *r, s.T, H, dk, dv, vp, nchunks, vt);
        }
        if (e != cudaSuccess) return e;
        const int64_t per = (int64_t)H * dk * (vp / 4);
        e = skn_launch_pdl(skn_ret_scan_kernel, dim3((unsigned)((per + 127) / 128), s.n_seqs), dim3(128), 0, st, 1, *r, s, r->state->d, H, dk, vp, nchunks);
        if (e != cudaSuccess) return e;
        if (tc) {
            e = cudaFuncSetAttribute(skn_ret_out_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
            if (e != cudaSuccess) return e;
            e = skn_launch_pdl(skn_ret_out_tc_kernel, ogrid, dim3(256), ret_out_tc_smem(dk, dv), st, 1, *r, s.T, H, dk, dv, vp, nchunks);
        } else {
            e = cudaFuncSetAttribute(skn_ret_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
            if (e != cudaSuccess) return e;
            e = skn_launch_pdl(skn_ret_out_kernel, ogrid, dim3(256), ret_out_smem(dv), st, 1, *r, s.T, H, dk, dv, vp, nchunks);
        }
    }
    return e;
}

// ---- angles and positions --------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(128)
skn_rot_table_kernel(skn_step st, const double *__restrict__ freq, int half, float2 *out, int ld) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int m = blockIdx.x, pos = st.pos[st.slot0 + m / st.T] + m % st.T;
    for (int i = threadIdx.x; i < half; i += 128) {
        // an fp32 product would be off by pos * 2^-24: the angle is formed and reduced in double
        const double a = (double)pos * freq[i], turns = rint(a * 0.15915494309189535);
        float s, c;
        sincosf((float)(a - turns * 6.283185307179586), &s, &c);
        out[(int64_t)m * ld + i] = make_float2(c, s);
    }
}

cudaError_t skn_launch_rot_table(const skn_step &s, const double *freq, int half, float2 *out, int ld, cudaStream_t st) {
    return skn_launch_pdl(skn_rot_table_kernel, dim3(s.n_seqs * s.T), dim3(128), 0, st, 1, s, freq, half, out, ld);
}

// Triggers no launch early: what follows it in the stream (the next step) starts when every launch before it is done, so a
// step's kernels may read what earlier steps left (states, caches) ahead of their own dependency wait.
__global__ void skn_advance_kernel(skn_step st, int32_t *pos, int32_t *status) {
    skn_pdl_wait();
    for (int s = threadIdx.x; s < st.n_seqs; s += blockDim.x) {
        const int p = pos[st.slot0 + s] + st.T;
        if (p > st.max_pos) atomicExch(status, SKN_ERR_SHAPE);
        pos[st.slot0 + s] = min(p, st.max_pos);
    }
}

cudaError_t skn_launch_advance(const skn_step &s, int32_t *pos, int32_t *status, cudaStream_t st) {
    return skn_launch_pdl(skn_advance_kernel, dim3(1), dim3(128), 0, st, 1, s, pos, status);
}

// ---- host-pointer forms ------------------------------------------------------------------------------------------------
namespace {
// carves 256-byte aligned pieces out of one allocation; first run with base NULL to measure
struct Arena {
    uint8_t *base;
    size_t used;
    template <class T> T *take(size_t n) {
        T *p = reinterpret_cast<T *>(base + used);
        used += (n * sizeof(T) + 255) / 256 * 256;
        return p;
    }
};
}

static int32_t upload(skn_ctx *ctx, void *dst, const void *src, size_t bytes) {
    SKN_CUDA(ctx, cudaMemcpyAsync(dst, src, bytes, cudaMemcpyHostToDevice, ctx->stream));
    return SKN_OK;
}

static int32_t check_step(skn_ctx *ctx, int32_t slots, int32_t seq0, int32_t n_seqs, int32_t T, const int32_t *pos, int32_t max_ctx) {
    if (seq0 < 0 || n_seqs < 1 || T < 1 || seq0 + n_seqs > slots || !pos) return skn_fail(ctx, SKN_ERR_ARG, "sequences outside the cache, or no positions");
    for (int s = 0; s < n_seqs; ++s)
        if (pos[s] < 0 || pos[s] + T > max_ctx) return skn_fail(ctx, SKN_ERR_SHAPE, "context of %d tokens exceeded", max_ctx);
    return SKN_OK;
}

void skn_rot_freqs(double base, int dims, double *out) {
    for (int i = 0; i < dims / 2; ++i) out[i] = pow(base, -2.0 * i / dims);
}

void skn_decay_powers(const double *decay, int heads, float *out) {
    for (int h = 0; h < heads; ++h)
        for (int n = 0; n <= SKN_RET_CHUNK; ++n) out[h * (SKN_RET_CHUNK + 1) + n] = (float)pow(decay[h], n);
}

int32_t skn_check_attn_spec(skn_ctx *ctx, const skn_attn_spec *a) {
    if (a->heads < 1 || a->kv_heads < 1 || a->dim < 1 || a->vdim < 1 || a->chunk < 0 || a->window < 0 || (a->chunk && a->window)) return skn_fail(ctx, SKN_ERR_ARG, "invalid attention geometry");
    if (a->heads % a->kv_heads || a->rot_dims < 0 || a->rot_dims % 2 || a->rot_dims > a->dim || a->dim > SKN_ATTN_MAX_DIM || a->vdim > SKN_ATTN_MAX_DIM)
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    return SKN_OK;
}

int32_t skn_check_retention_spec(skn_ctx *ctx, const skn_retention_spec *r) {
    if (r->heads < 1 || r->dim < 1 || r->vdim < 1 || !r->decay) return skn_fail(ctx, SKN_ERR_ARG, "invalid retention geometry");
    if (r->rot_dims < 0 || r->rot_dims % 2 || r->rot_dims > r->dim || r->dim > SKN_ATTN_MAX_DIM || r->vdim > SKN_ATTN_MAX_DIM)
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    return SKN_OK;
}

extern "C" {

int32_t skn_chunk_attn(skn_kvcache *kv, const skn_attn_spec *spec, int32_t seq0, int32_t n_seqs, int32_t T, const int32_t *pos_host,
                       int32_t max_ctx, const float *q_gain_host, const float *k_gain_host, const float *q_host, const float *k_host,
                       const float *v_host, const float *sink_host, float *out_host) {
    if (!skn_kv_ok(kv) || !kv->by_position) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "not a position-addressed cache");
    skn_ctx *ctx = kv->ctx;
    SKN_ENTER(ctx);
    if (!spec || !q_host || !k_host || !v_host || !out_host || !q_gain_host != !k_gain_host) return skn_fail(ctx, SKN_ERR_ARG, "NULL argument");
    int32_t rc = skn_check_attn_spec(ctx, spec);
    if (rc) return rc;
    if (spec->kv_heads != kv->n_kv_heads || spec->dim != kv->head_dim || spec->vdim != kv->v_dim) return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    if ((rc = check_step(ctx, kv->batch, seq0, n_seqs, T, pos_host, max_ctx))) return rc;
    const int span = spec->chunk > 0 ? spec->chunk : spec->window;
    const int need = span > 0 && span + T < max_ctx ? span + T : max_ctx;
    if (kv->capacity < need) return skn_fail(ctx, SKN_ERR_SHAPE, "this step needs a cache of %d tokens", need);
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    const int H = spec->heads, G = spec->kv_heads, D = spec->dim, V = spec->vdim, M = n_seqs * T, half = spec->rot_dims / 2;
    float *q, *out, *scratch, *qg, *kg, *sink;
    int32_t *pos;
    unsigned *tickets;
    float2 *rot;
    double *freq;
    __nv_bfloat16 *q16;
    const size_t nscr = skn_attn_scratch(M, H, V, span, max_ctx);
    Arena a = {nullptr, 0};
    for (int pass = 0; pass < 2; ++pass) {
        q = a.take<float>((size_t)M * ((size_t)H * D + (size_t)G * (D + V)));
        out = a.take<float>((size_t)M * H * V); scratch = a.take<float>(nscr); qg = a.take<float>(D); kg = a.take<float>(D); sink = a.take<float>(H);
        pos = a.take<int32_t>(kv->batch); tickets = a.take<unsigned>((size_t)M * H); rot = a.take<float2>((size_t)M * (half + 1));
        freq = a.take<double>(half + 1); q16 = a.take<__nv_bfloat16>((size_t)M * H * kv->k_pitch);
        if (pass == 0) {
            if ((rc = skn_stage_reserve(ctx, &ctx->d_scratch, &ctx->d_scratch_bytes, a.used))) return rc;
            a.base = (uint8_t *)ctx->d_scratch;
            a.used = 0;
        }
    }
    double hf[SKN_ATTN_MAX_DIM / 2 + 1];
    skn_rot_freqs(spec->rot_base, spec->rot_dims, hf);
    if ((rc = upload(ctx, pos + seq0, pos_host, sizeof(int32_t) * n_seqs)) || (rc = upload(ctx, freq, hf, sizeof(double) * half))) return rc;
    if (q_gain_host && ((rc = upload(ctx, qg, q_gain_host, sizeof(float) * D)) || (rc = upload(ctx, kg, k_gain_host, sizeof(float) * D)))) return rc;
    if (sink_host && (rc = upload(ctx, sink, sink_host, sizeof(float) * H))) return rc;
    SKN_CUDA(ctx, cudaMemsetAsync(tickets, 0, (size_t)M * H * sizeof(unsigned), ctx->stream));
    // joint rows [q | k | v], as the projection of a decoder leaves them
    const int64_t ld = (int64_t)H * D + (int64_t)G * (D + V);
    SKN_CUDA(ctx, cudaMemcpy2DAsync(q, ld * 4, q_host, (size_t)H * D * 4, (size_t)H * D * 4, M, cudaMemcpyHostToDevice, ctx->stream));
    SKN_CUDA(ctx, cudaMemcpy2DAsync(q + H * D, ld * 4, k_host, (size_t)G * D * 4, (size_t)G * D * 4, M, cudaMemcpyHostToDevice, ctx->stream));
    SKN_CUDA(ctx, cudaMemcpy2DAsync(q + H * D + G * D, ld * 4, v_host, (size_t)G * V * 4, (size_t)G * V * 4, M, cudaMemcpyHostToDevice, ctx->stream));
    const skn_step st = {seq0, n_seqs, T, pos, max_ctx};
    if (half) SKN_CUDA(ctx, skn_launch_rot_table(st, freq, half, rot, half, ctx->stream));
    skn_attn_args x = {};
    x.kv = kv; x.heads = H; x.chunk = spec->chunk; x.window = spec->window; x.sink = sink_host ? sink : nullptr; x.scale = spec->scale; x.softcap = spec->softcap; x.eps = spec->eps;
    x.q_gain = q_gain_host ? qg : nullptr; x.k_gain = q_gain_host ? kg : nullptr;
    x.rot = skn_rot{rot, half, half};
    x.q = q; x.k = q + H * D; x.v = q + H * D + G * D; x.ld = ld;
    x.out_scale = 1.f; x.out = skn_rows_out{out, (int64_t)H * V, nullptr, 0};
    x.scratch = scratch; x.tickets = tickets; x.q16 = q16;
    SKN_CUDA(ctx, T == 1 ? skn_launch_mix_decode(ctx, st, &x, nullptr, ctx->stream) : skn_launch_mix_prefill(ctx, st, &x, nullptr, ctx->stream));
    SKN_CUDA(ctx, cudaMemcpyAsync(out_host, out, (size_t)M * H * V * 4, cudaMemcpyDeviceToHost, ctx->stream));
    return skn_sync(ctx);
}

int32_t skn_retention(skn_state *s, const skn_retention_spec *spec, int32_t seq0, int32_t n_seqs, int32_t T, const int32_t *pos_host,
                      int32_t max_ctx, const float *q_host, const float *k_host, const float *v_host, const float *g_host, float *out_host) {
    if (!s || s->magic != SKN_MAGIC_STATE || !skn_ctx_ok(s->ctx)) return skn_fail(nullptr, SKN_ERR_BAD_HANDLE, "bad state handle");
    skn_ctx *ctx = s->ctx;
    SKN_ENTER(ctx);
    if (!spec || !q_host || !k_host || !v_host || !g_host || !out_host) return skn_fail(ctx, SKN_ERR_ARG, "NULL argument");
    int32_t rc = skn_check_retention_spec(ctx, spec);
    if (rc) return rc;
    if (spec->heads != s->heads || spec->dim != s->k_dim || spec->vdim != s->v_dim) return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    if ((rc = check_step(ctx, s->slots, seq0, n_seqs, T, pos_host, max_ctx))) return rc;
    SKN_CUDA(ctx, cudaSetDevice(ctx->device));
    const int H = spec->heads, D = spec->dim, V = spec->vdim, M = n_seqs * T, half = spec->rot_dims / 2, nch = (T + SKN_RET_CHUNK - 1) / SKN_RET_CHUNK;
    const int64_t ld = (int64_t)H * (2 * D + 2 * V);
    float *rows, *out, *pw, *chunks;
    int32_t *pos;
    float2 *rot;
    double *freq;
    Arena a = {nullptr, 0};
    for (int pass = 0; pass < 2; ++pass) {
        rows = a.take<float>((size_t)M * ld); out = a.take<float>((size_t)M * H * V); pw = a.take<float>((size_t)H * (SKN_RET_CHUNK + 1));
        chunks = a.take<float>((size_t)n_seqs * nch * H * D * s->v_pitch); pos = a.take<int32_t>(s->slots);
        rot = a.take<float2>((size_t)M * (half + 1)); freq = a.take<double>(half + 1);
        if (pass == 0) {
            if ((rc = skn_stage_reserve(ctx, &ctx->d_scratch, &ctx->d_scratch_bytes, a.used))) return rc;
            a.base = (uint8_t *)ctx->d_scratch;
            a.used = 0;
        }
    }
    double hf[SKN_ATTN_MAX_DIM / 2 + 1];
    skn_rot_freqs(spec->rot_base, spec->rot_dims, hf);
    float *hp = (float *)malloc((size_t)H * (SKN_RET_CHUNK + 1) * sizeof(float));
    if (!hp) return skn_fail(ctx, SKN_ERR_OOM, "host allocation failed");
    skn_decay_powers(spec->decay, H, hp);
    rc = upload(ctx, pw, hp, (size_t)H * (SKN_RET_CHUNK + 1) * sizeof(float));
    cudaStreamSynchronize(ctx->stream);
    free(hp);
    if (rc || (rc = upload(ctx, pos + seq0, pos_host, sizeof(int32_t) * n_seqs)) || (rc = upload(ctx, freq, hf, sizeof(double) * half))) return rc;
    const float *src[4] = {q_host, k_host, v_host, g_host};
    const size_t w[4] = {(size_t)H * D, (size_t)H * D, (size_t)H * V, (size_t)H * V};
    float *dst = rows;
    for (int i = 0; i < 4; ++i) {
        SKN_CUDA(ctx, cudaMemcpy2DAsync(dst, ld * 4, src[i], w[i] * 4, w[i] * 4, M, cudaMemcpyHostToDevice, ctx->stream));
        dst += w[i];
    }
    const skn_step st = {seq0, n_seqs, T, pos, max_ctx};
    if (half) SKN_CUDA(ctx, skn_launch_rot_table(st, freq, half, rot, half, ctx->stream));
    skn_ret_args x = {};
    x.state = s; x.eps = spec->eps; x.rot = skn_rot{rot, half, half}; x.k_scale = (float)(1.0 / sqrt((double)D)); x.powers = pw;
    x.q = rows; x.k = rows + w[0]; x.v = rows + 2 * w[0]; x.g = rows + 2 * w[0] + w[2]; x.ld = ld;
    x.out_scale = 1.f; x.out = skn_rows_out{out, (int64_t)H * V, nullptr, 0}; x.exact = spec->exact != 0; x.chunks = chunks;
    SKN_CUDA(ctx, T == 1 ? skn_launch_mix_decode(ctx, st, nullptr, &x, ctx->stream) : skn_launch_mix_prefill(ctx, st, nullptr, &x, ctx->stream));
    SKN_CUDA(ctx, cudaMemcpyAsync(out_host, out, (size_t)M * H * V * 4, cudaMemcpyDeviceToHost, ctx->stream));
    return skn_sync(ctx);
}

}  // extern "C"
