// Latent attention (see skn_latent.cuh).
#include "skn_latent.cuh"
#include "skn_ptx.cuh"

#include <math.h>

constexpr int LT = 256;                  // threads
constexpr int QL_COLS = 128;             // latent columns of a CTA of the absorbed query kernel
constexpr int OL_ROWS = 32;              // value rows of a CTA of the absorbed output kernel

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

// out[m][h][v] = sigmoid(gate) * (W_uv row (h, v) . ol[m][h]).  CTA: OL_ROWS rows of one head, RB tokens.  smem (floats): ol [RB][kvp]
template <int RB>
__global__ void __launch_bounds__(LT)
skn_latent_out_kernel(skn_latent_args a, const uint8_t *__restrict__ ukv, int64_t wpitch, int row_tiles, int M) {
    extern __shared__ __align__(16) float sm[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, m0 = blockIdx.y * RB;
    const int h = blockIdx.x / row_tiles, v0 = (blockIdx.x % row_tiles) * OL_ROWS, v1 = min(a.vdim, v0 + OL_ROWS);
    const uint8_t *w = ukv + ((int64_t)a.heads * a.dim + (int64_t)h * a.vdim) * wpitch;
    for (int v = v0 + warp; v < v1; v += LT / 32)
        for (int64_t i = (int64_t)lane * 128; i < wpitch; i += 32 * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(w + v * wpitch + i));
    skn_pdl_wait();
    for (int i = tid; i < RB * a.kvp; i += LT) {
        const int r = i / a.kvp, k = i % a.kvp;
        sm[i] = m0 + r < M ? __ldcg(a.ol + ((int64_t)(m0 + r) * a.heads + h) * a.kvp + k) : 0.f;
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
            for (int r = 0; r < RB; ++r)
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[x][r] = fmaf(sm[r * a.kvp + k + e], f[e], acc[x][r]);
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

cudaError_t skn_launch_latent_absorbed(const skn_step &s, const skn_latent_args &a, bool append, cudaStream_t st) {
    const int M = s.n_seqs * s.T;
    const bool bf = a.kv->dtype == SKN_KV_BF16;
    cudaError_t e = M == 1 ? (bf ? launch_q<__nv_bfloat16, 1>(s, a, append, st) : launch_q<float, 1>(s, a, append, st))
                           : (bf ? launch_q<__nv_bfloat16, 2>(s, a, append, st) : launch_q<float, 2>(s, a, append, st));
    if (e != cudaSuccess) return e;
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
    if ((e = skn_launch_attn_rows(s, x, st)) != cudaSuccess) return e;
    const int row_tiles = (a.vdim + OL_ROWS - 1) / OL_ROWS;
    const uint8_t *w = (const uint8_t *)a.ukv->d_blocks;
    if (M == 1)
        return skn_launch_pdl(skn_latent_out_kernel<1>, dim3(a.heads * row_tiles, 1), dim3(LT), (size_t)a.kvp * 4, st, 1, a, w, a.ukv->pitch, row_tiles, M);
    return skn_launch_pdl(skn_latent_out_kernel<4>, dim3(a.heads * row_tiles, (M + 3) / 4), dim3(LT), (size_t)4 * a.kvp * 4, st, 1, a, w, a.ukv->pitch, row_tiles, M);
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
