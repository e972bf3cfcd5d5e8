// Selective state space (see skn_ssm.cuh).
//
//  skn_ssm_step_kernel    tokens one after the other, state in registers; a CTA owns one head of one sequence (64 of its columns).  One
//                         token per sequence is the decode step; the fp32 decoder and short portions run any number
//  skn_ssm_conv_kernel    many tokens: convolution and silu of every channel (bf16 rows), step sizes and log decays
//  skn_ssm_chunk_kernel   what a chunk adds to the state: sum over its tokens j of exp(cum_end - cum_j) dt_j B_j x_j^T
//  skn_ssm_scan_kernel    states at the chunk starts and after the step; files the convolution's last inputs
//  skn_ssm_out_kernel     y_i = sum_{j <= i} exp(cum_i - cum_j) dt_j (C_i . B_j) x_j + exp(cum_i) S^T C_i + D x_i, times silu(z)
//
// In the chunk kernels x, B and C are bf16 and enter the tensor cores exactly, sums are fp32.  What is added to the state enters as three bf16
// terms (24 bits); in the outputs, which only read the state, weights and states enter as two (16 bits), as softmax weights do.
#include "skn_ssm.cuh"
#include "skn_mma.cuh"

#include <math.h>

constexpr int SC = SKN_SSM_CHUNK;
constexpr int STEP_THREADS = 256, STEP_COLS = 64;

__device__ __forceinline__ float ssm_silu(float v) { return v / (1.f + expf(-v)); }
// relative error a few 1e-7: where the result is rounded to bf16 or many are formed
__device__ __forceinline__ float ssm_silu_fast(float v) { return __fdividef(v, 1.f + __expf(fminf(-v, 80.f))); }
__device__ __forceinline__ float ssm_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// convolution and silu of channel c at token t of a sequence whose rows start at `rows` and that had p0 tokens before
__device__ __forceinline__ float ssm_channel(const skn_ssm_args &a, const float *rows, const float *ring, int channels, int p0, int t, int c) {
    float v = a.conv_b[c];
    for (int k = 0; k < a.taps; ++k) {
        const int back = t - (a.taps - 1) + k;
        float u = 0.f;
        if (back >= 0) u = __ldcg(rows + back * a.ld + c);
        else if (p0 + back >= 0) u = __ldcg(ring + (int64_t)((p0 + back) % a.taps) * channels + c);
        v = fmaf(a.conv[(int64_t)k * channels + c], u, v);
    }
    return ssm_silu(v);
}

// smem (floats): x [STEP_COLS] | B [np] | C [np] | o [STEP_THREADS * 4]
template <int RPT>
__global__ void __launch_bounds__(STEP_THREADS)
skn_ssm_step_kernel(skn_ssm_args a, skn_step st, float *S_, float *ring_, int ring_pitch, int slices) {
    extern __shared__ __align__(16) float sm[];
    // (no early trigger: see skn_mix_decode_kernel)
    const int tid = threadIdx.x, seq = blockIdx.y, slot = st.slot0 + seq;
    if ((int)blockIdx.x >= a.heads * slices) {
        skn_pdl_wait();
        if (tid < 32)
            for (int t = 0; t < st.T; ++t) skn_route_row(a.route, (int64_t)seq * st.T + t, sm);
        return;
    }
    const int h = blockIdx.x / slices, c0 = (blockIdx.x % slices) * STEP_COLS, vs = min(STEP_COLS, a.vp - c0);
    const int nv = vs / 4, lanes = STEP_THREADS / nv, cg = tid % nv, rl = tid / nv;
    const int per_group = a.heads / a.groups, g = h / per_group;
    float *xs = sm, *bs = xs + STEP_COLS, *cs = bs + a.np, *red = cs + a.np;
    float *S = S_ + (((int64_t)slot * a.heads + h) * a.np) * a.vp + c0 + cg * 4;
    // the state depends on earlier steps only
    float4 s[RPT];
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const int i = rl + r * lanes;
        s[r] = rl < lanes && i < a.np ? __ldcg(reinterpret_cast<const float4 *>(S + (int64_t)i * a.vp)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int inner = a.heads * a.vp, channels = skn_ssm_channels(a.heads, a.vp, a.groups, a.np);
    const float av = a.a[h], bias = a.dt_bias[h], dv = a.d[h];
    float *ring = ring_ + (int64_t)slot * a.taps * ring_pitch;
    skn_pdl_wait();
    const int p0 = st.pos[slot];
    if (p0 == 0)
#pragma unroll
        for (int r = 0; r < RPT; ++r) s[r] = make_float4(0.f, 0.f, 0.f, 0.f);
    const float *row0 = a.proj + (int64_t)seq * st.T * a.ld, *xbc = row0 + inner;
    const int xc = h * a.vp + c0, bc = inner + g * a.np, cc = bc + a.groups * a.np;
    const bool fold = nv <= 32 && 32 % nv == 0;
    for (int t = 0; t < st.T; ++t) {
        for (int i = tid; i < vs + 2 * a.np; i += STEP_THREADS) {
            const int c = i < vs ? xc + i : i < vs + a.np ? bc + i - vs : cc + i - vs - a.np;
            const float v = ssm_channel(a, xbc, ring, ring_pitch, p0, t, c);
            if (i < vs) xs[i] = v;
            else bs[i - vs] = v;                     // (B, then C behind it)
        }
        const float dt = ssm_softplus(__ldcg(row0 + (int64_t)t * a.ld + inner + channels + h) + bias), decay = expf(av * dt);
        __syncthreads();
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        if (rl < lanes) {
            const float4 x = *reinterpret_cast<const float4 *>(xs + cg * 4);
#pragma unroll
            for (int r = 0; r < RPT; ++r) {
                const int i = rl + r * lanes;
                if (i >= a.np) continue;
                const float k = dt * bs[i], q = cs[i];
                s[r].x = fmaf(decay, s[r].x, k * x.x);
                s[r].y = fmaf(decay, s[r].y, k * x.y);
                s[r].z = fmaf(decay, s[r].z, k * x.z);
                s[r].w = fmaf(decay, s[r].w, k * x.w);
                o.x = fmaf(q, s[r].x, o.x);
                o.y = fmaf(q, s[r].y, o.y);
                o.z = fmaf(q, s[r].z, o.z);
                o.w = fmaf(q, s[r].w, o.w);
            }
        }
        // sums over the rows: first across the lanes of a warp that hold the same columns
        int parts = min(lanes, a.np);
        if (fold) {
            for (int d = nv; d < 32; d <<= 1) {
                o.x += __shfl_xor_sync(0xffffffffu, o.x, d);
                o.y += __shfl_xor_sync(0xffffffffu, o.y, d);
                o.z += __shfl_xor_sync(0xffffffffu, o.z, d);
                o.w += __shfl_xor_sync(0xffffffffu, o.w, d);
            }
            parts = STEP_THREADS / 32;
            if ((tid & 31) < nv) *reinterpret_cast<float4 *>(red + ((tid >> 5) * nv + cg) * 4) = o;
        } else if (rl < lanes) {
            *reinterpret_cast<float4 *>(red + (rl * nv + cg) * 4) = o;
        }
        __syncthreads();
        if (tid < vs) {
            float y = dv * xs[tid];
            for (int p = 0; p < parts; ++p) y += red[p * vs + tid];
            const float z = __ldcg(row0 + (int64_t)t * a.ld + xc + tid);
            a.y[((int64_t)seq * st.T + t) * a.ld_y + xc + tid] = y * ssm_silu(z);
        }
        if (t + 1 < st.T) __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const int i = rl + r * lanes;
        if (rl < lanes && i < a.np) *reinterpret_cast<float4 *>(S + (int64_t)i * a.vp) = s[r];
    }
    if (st.T == 1) {
        // this token's inputs: x by its own CTA, B and C by the first of the group's
        float *dst = ring + (int64_t)(p0 % a.taps) * ring_pitch;
        for (int i = tid; i < vs; i += STEP_THREADS) dst[xc + i] = __ldcg(xbc + xc + i);
        if (h % per_group == 0 && c0 == 0)
            for (int i = tid; i < 2 * a.np; i += STEP_THREADS) {
                const int c = i < a.np ? bc + i : cc + i - a.np;
                dst[c] = __ldcg(xbc + c);
            }
    }
}

// files the convolution's inputs of the step's last taps - 1 tokens; thread i of the sequence's n
__device__ __forceinline__ void ssm_file_inputs(const skn_ssm_args &a, const skn_step &st, float *ring_, int ring_pitch, int seq, int64_t i) {
    const int channels = skn_ssm_channels(a.heads, a.vp, a.groups, a.np), inner = a.heads * a.vp;
    const int back = (int)(i / channels) + 1, c = (int)(i % channels), t = st.T - back;
    if (back >= a.taps || t < 0) return;
    const int slot = st.slot0 + seq, p = st.pos[slot] + t;
    ring_[((int64_t)slot * a.taps + p % a.taps) * ring_pitch + c] = __ldcg(a.proj + ((int64_t)seq * st.T + t) * a.ld + inner + c);
}

__global__ void __launch_bounds__(256)
skn_ssm_file_kernel(skn_ssm_args a, skn_step st, float *ring, int ring_pitch) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    ssm_file_inputs(a, st, ring, ring_pitch, blockIdx.y, (int64_t)blockIdx.x * 256 + threadIdx.x);
}

template <int RPT>
static cudaError_t launch_step(const skn_step &s, const skn_ssm_args &a, int slices, cudaStream_t st) {
    const size_t own = ((size_t)STEP_COLS + 2 * a.np + STEP_THREADS * 4) * sizeof(float), rt = skn_route_smem(a.route);
    const dim3 grid(a.heads * slices + (a.route.logits ? 1 : 0), s.n_seqs);
    return skn_launch_pdl(skn_ssm_step_kernel<RPT>, grid, dim3(STEP_THREADS), own > rt ? own : rt, st, 1, a, s, a.state->d, a.ring->d, a.ring->v_pitch, slices);
}

cudaError_t skn_launch_ssm_step(const skn_step &s, const skn_ssm_args &a, cudaStream_t st) {
    const int slices = (a.vp + STEP_COLS - 1) / STEP_COLS, widest = a.vp < STEP_COLS ? a.vp : STEP_COLS;
    const int lanes = STEP_THREADS / (widest / 4), rpt = (a.np + lanes - 1) / lanes;
    cudaError_t e = rpt <= 1 ? launch_step<1>(s, a, slices, st) : rpt <= 2 ? launch_step<2>(s, a, slices, st) : rpt <= 4 ? launch_step<4>(s, a, slices, st)
                    : rpt <= 8 ? launch_step<8>(s, a, slices, st) : rpt <= 16 ? launch_step<16>(s, a, slices, st)
                    : rpt <= 32 ? launch_step<32>(s, a, slices, st) : cudaErrorNotSupported;
    if (e != cudaSuccess || s.T == 1 || a.taps == 1) return e;
    const int64_t n = (int64_t)(a.taps - 1) * skn_ssm_channels(a.heads, a.vp, a.groups, a.np);
    return skn_launch_pdl(skn_ssm_file_kernel, dim3((unsigned)((n + 255) / 256), s.n_seqs), dim3(256), 0, st, 1, a, s, a.ring->d, a.ring->v_pitch);
}

// ---- many tokens -----------------------------------------------------------------------------------------------------
constexpr int CV_TOKENS = 16;               // tokens of a thread's run

// CTA x below `tiles`: four channels per thread, CV_TOKENS tokens; beyond: step sizes and log decays of one chunk
template <int TAPS>
__global__ void __launch_bounds__(128)
skn_ssm_conv_kernel(skn_ssm_args a, skn_step st, const float *ring_, int ring_pitch, int tiles) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int seq = blockIdx.z, slot = st.slot0 + seq, p0 = st.pos[slot], inner = a.heads * a.vp;
    const int channels = skn_ssm_channels(a.heads, a.vp, a.groups, a.np);
    const float *row0 = a.proj + (int64_t)seq * st.T * a.ld;
    if ((int)blockIdx.x >= tiles) {
        // one chunk, 32 heads: a warp takes a quarter of the tokens, a lane one head
        const int t0 = blockIdx.y * CV_TOKENS, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
        if (t0 % SC) return;
        __shared__ float quarter[4][32];
        const int h = ((int)blockIdx.x - tiles) * 32 + lane, first = t0 + warp * (SC / 4);
        const bool in = h < a.heads;
        const float av = in ? a.a[h] : 0.f, bias = in ? a.dt_bias[h] : 0.f;
        float dt[SC / 4], sum = 0.f;
#pragma unroll
        for (int i = 0; i < SC / 4; ++i) dt[i] = in && first + i < st.T ? __ldcg(row0 + (int64_t)(first + i) * a.ld + inner + channels + h) : 0.f;
#pragma unroll
        for (int i = 0; i < SC / 4; ++i) {
            dt[i] = ssm_softplus(dt[i] + bias);
            sum += dt[i];
        }
        quarter[warp][lane] = sum;
        __syncthreads();
        float cum = 0.f;
        for (int w = 0; w < warp; ++w) cum += quarter[w][lane];
#pragma unroll
        for (int i = 0; i < SC / 4; ++i) {
            cum += dt[i];
            if (!in || first + i >= st.T) continue;
            const int64_t at = ((int64_t)seq * st.T + first + i) * a.heads + h;
            a.dt[at] = dt[i];
            a.cum[at] = av * cum;
        }
        return;
    }
    const int c = (blockIdx.x * 128 + threadIdx.x) * 4;
    if (c >= channels) return;
    const float *in = row0 + inner + c, *ring = ring_ + (int64_t)slot * a.taps * ring_pitch + c;
    auto load = [&](int t) {
        if (t >= 0) return __ldcg(reinterpret_cast<const float4 *>(in + (int64_t)t * a.ld));
        if (p0 + t >= 0) return __ldcg(reinterpret_cast<const float4 *>(ring + (int64_t)((p0 + t) % a.taps) * ring_pitch));
        return make_float4(0.f, 0.f, 0.f, 0.f);
    };
    const float4 b = __ldg(reinterpret_cast<const float4 *>(a.conv_b + c));
    const int t0 = blockIdx.y * CV_TOKENS, t1 = min(st.T, t0 + CV_TOKENS);
    __nv_bfloat16 *out = a.xbc + (int64_t)seq * st.T * channels + c;
    auto put = [&](int t, float4 v) {
        uint2 w;
        w.x = pack_bf16(ssm_silu_fast(v.x), ssm_silu_fast(v.y));
        w.y = pack_bf16(ssm_silu_fast(v.z), ssm_silu_fast(v.w));
        *reinterpret_cast<uint2 *>(out + (int64_t)t * channels) = w;
    };
    auto fma4 = [](const float4 &w, const float4 &u, float4 v) {
        v.x = fmaf(w.x, u.x, v.x); v.y = fmaf(w.y, u.y, v.y); v.z = fmaf(w.z, u.z, v.z); v.w = fmaf(w.w, u.w, v.w);
        return v;
    };
    if constexpr (TAPS > 0) {
        // every input of the run is loaded before the first output is stored
        float4 w[TAPS], u[CV_TOKENS + TAPS - 1];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) w[k] = __ldg(reinterpret_cast<const float4 *>(a.conv + (int64_t)k * channels + c));
#pragma unroll
        for (int i = 0; i < CV_TOKENS + TAPS - 1; ++i) {
            const int t = t0 - (TAPS - 1) + i;
            u[i] = t < t1 ? load(t) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < CV_TOKENS; ++i) {
            float4 v = b;
#pragma unroll
            for (int k = 0; k < TAPS; ++k) v = fma4(w[k], u[i + k], v);
            if (t0 + i < t1) put(t0 + i, v);
        }
    } else {
        for (int t = t0; t < t1; ++t) {
            float4 v = b;
            for (int k = 0; k < a.taps; ++k) v = fma4(__ldg(reinterpret_cast<const float4 *>(a.conv + (int64_t)k * channels + c)), load(t - (a.taps - 1) + k), v);
            put(t, v);
        }
    }
}

// rows of a chunk in shared memory: `cols` valid columns (a multiple of 8) of src, zero beyond, row stride `stride`.  A warp takes a row.
__device__ __forceinline__ void ssm_load_rows(__nv_bfloat16 *dst, int stride, const __nv_bfloat16 *src, int64_t ld, int L, int cols, int wide) {
    const int lane = threadIdx.x & 31;
    for (int t = threadIdx.x >> 5; t < SC; t += 4)
        for (int c = lane * 8; c < wide; c += 256) {
            const bool in = t < L && c < cols;
            cp_async16(skn_smem_u32(dst + t * stride + c), in ? src + t * ld + c : src, in);
        }
}
// the same for rows of DV columns, DV / 8 threads to a row: row n at src + n * ld for n < valid
template <int DV>
__device__ __forceinline__ void ssm_load_tile(__nv_bfloat16 *dst, const __nv_bfloat16 *src, int64_t ld, int rows, int valid, int cols) {
    constexpr int TPR = DV / 8;
    const int c = threadIdx.x % TPR * 8;
    for (int n = threadIdx.x / TPR; n < rows; n += 128 / TPR) {
        const bool in = n < valid && c < cols;
        cp_async16(skn_smem_u32(dst + n * (DV + 8) + c), in ? src + n * ld + c : src, in);
    }
}

// the first N bf16 terms of (a, b), packed
template <int N>
__device__ __forceinline__ void bf16_terms(float a, float b, uint32_t (&o)[N]) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
        o[i] = pack_bf16(a, b);
        if (i + 1 < N) less_bf16(a, b, o[i]);
    }
}

__host__ __device__ constexpr int up16(int n) { return (n + 15) / 16 * 16; }

// smem (bf16): B [SC][np16 + 8] | weighted x, three terms [3][SC][DV + 8]
static size_t ssm_chunk_smem(int np, int DV) { return ((size_t)SC * (up16(np) + 8) + (size_t)3 * SC * (DV + 8)) * 2; }

// CTA: `per` heads of one group
template <int DV>
__global__ void __launch_bounds__(128)
skn_ssm_chunk_kernel(skn_ssm_args a, int T, int nchunks, int per) {
    extern __shared__ __align__(16) uint8_t smb[];
    __shared__ float wj[SC];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int np16 = up16(a.np), bs = np16 + 8, xs = DV + 8;
    __nv_bfloat16 *B = reinterpret_cast<__nv_bfloat16 *>(smb), *X = B + SC * bs;
    const int c = blockIdx.x, h0 = blockIdx.y * per, seq = blockIdx.z, t0 = c * SC, L = min(SC, T - t0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int channels = skn_ssm_channels(a.heads, a.vp, a.groups, a.np), inner = a.heads * a.vp, g = h0 / (a.heads / a.groups);
    const int64_t row0 = (int64_t)seq * T + t0;
    const __nv_bfloat16 *rows = a.xbc + row0 * channels;
    ssm_load_rows(B, bs, rows + inner + g * a.np, channels, L, a.np, np16);
    asm volatile("cp.async.commit_group;" ::: "memory");
    // a head's x: PX pieces of 8 elements per thread, fetched while the head before is multiplied
    constexpr int PX = SC * (DV / 8) / 128;
    uint4 pre[PX];
    auto fetch = [&](int h) {
#pragma unroll
        for (int i = 0; i < PX; ++i) {
            const int at = tid + i * 128, t = at / (DV / 8), v = at % (DV / 8) * 8;
            pre[i] = t < L && v < a.vp ? __ldcg(reinterpret_cast<const uint4 *>(rows + (int64_t)t * channels + h * a.vp + v)) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    fetch(h0);
    for (int h = h0; h < h0 + per; ++h) {
        if (tid < SC) wj[tid] = tid < L ? __expf(a.cum[(row0 + L - 1) * a.heads + h] - a.cum[(row0 + tid) * a.heads + h]) * a.dt[(row0 + tid) * a.heads + h] : 0.f;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
#pragma unroll
        for (int i = 0; i < PX; ++i) {
            const int at = tid + i * 128, t = at / (DV / 8), v = at % (DV / 8) * 8;
            const uint32_t in[4] = {pre[i].x, pre[i].y, pre[i].z, pre[i].w};
            const float w = wj[t];
            uint32_t o[4][3];
#pragma unroll
            for (int e = 0; e < 4; ++e) bf16_terms<3>(__uint_as_float(in[e] << 16) * w, __uint_as_float(in[e] & 0xFFFF0000u) * w, o[e]);
#pragma unroll
            for (int x = 0; x < 3; ++x) *reinterpret_cast<uint4 *>(X + ((size_t)x * SC + t) * xs + v) = make_uint4(o[0][x], o[1][x], o[2][x], o[3][x]);
        }
        __syncthreads();
        if (h + 1 < h0 + per) fetch(h + 1);
        float *out = a.chunks + ((((int64_t)seq * nchunks + c) * a.heads + h) * a.np) * a.vp;
        for (int mt = warp; mt < np16 / 16; mt += 4) {
            float acc[DV / 8][4];
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
            for (int kk = 0; kk < SC; kk += 16) {
                uint32_t af[4];                  // B^T: rows n, columns j
                ldsm4t(af, skn_smem_u32(B + (size_t)(kk + (lane & 7) + (lane >> 4) * 8) * bs + mt * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
                for (int x = 2; x >= 0; --x)
#pragma unroll
                    for (int n = 0; n < DV / 16; ++n) {
                        uint32_t bf[4];
                        ldsm4t(bf, skn_smem_u32(X + ((size_t)x * SC + kk + (lane & 7) + ((lane >> 3) & 1) * 8) * xs + n * 16 + (lane >> 4) * 8));
                        mma_bf16(acc[2 * n], af, bf[0], bf[1]);
                        mma_bf16(acc[2 * n + 1], af, bf[2], bf[3]);
                    }
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int n = mt * 16 + (lane >> 2) + e * 8;
                if (n >= a.np) continue;
#pragma unroll
                for (int i = 0; i < DV / 8; ++i) {
                    const int v = i * 8 + (lane & 3) * 2;
                    if (v < a.vp) *reinterpret_cast<float2 *>(out + (int64_t)n * a.vp + v) = make_float2(acc[i][2 * e], acc[i][2 * e + 1]);
                }
            }
        }
        __syncthreads();
    }
}

// chunk sums -> states at the chunk starts (two bf16 terms), and the state after the step; CTAs from `blocks` on file the convolution's inputs
__global__ void __launch_bounds__(128)
skn_ssm_scan_kernel(skn_ssm_args a, skn_step st, float *S_, float *ring, int ring_pitch, int nchunks, int blocks) {
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int seq = blockIdx.y, slot = st.slot0 + seq, T = st.T;
    if ((int)blockIdx.x >= blocks) {
        ssm_file_inputs(a, st, ring, ring_pitch, seq, (int64_t)((int)blockIdx.x - blocks) * 128 + threadIdx.x);
        return;
    }
    const int64_t head = (int64_t)a.np * (a.vp / 4), per = a.heads * head, i = (int64_t)blockIdx.x * 128 + threadIdx.x;
    if (i >= per) return;
    const int h = (int)(i / head);
    const float4 *p = reinterpret_cast<const float4 *>(a.chunks) + (int64_t)seq * nchunks * per + i;
    // term planes [np][vp] of a head behind one another
    uint2 *start = reinterpret_cast<uint2 *>(a.starts) + ((int64_t)seq * nchunks * a.heads + h) * 2 * head + i % head;
    float4 *sp = reinterpret_cast<float4 *>(S_) + (int64_t)slot * per + i;
    float4 s = st.pos[slot] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *sp;
    const float *cum = a.cum + (int64_t)seq * T * a.heads + h;
    for (int c0 = 0; c0 < nchunks; c0 += 8) {
        float4 v[8];
        float d[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (c0 + u < nchunks) {
                v[u] = __ldcg(p + (int64_t)(c0 + u) * per);
                d[u] = cum[(int64_t)(min(T, (c0 + u + 1) * SC) - 1) * a.heads];
            }
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (c0 + u < nchunks) {
                uint32_t lo[2], hi[2];
                bf16_terms<2>(s.x, s.y, lo);
                bf16_terms<2>(s.z, s.w, hi);
                uint2 *q = start + (int64_t)(c0 + u) * per * 2;
                __stcg(q, make_uint2(lo[0], hi[0]));
                __stcg(q + head, make_uint2(lo[1], hi[1]));
                const float f = __expf(d[u]);
                s = make_float4(fmaf(f, s.x, v[u].x), fmaf(f, s.y, v[u].y), fmaf(f, s.z, v[u].z), fmaf(f, s.w, v[u].w));
            }
    }
    *sp = s;
}

// smem (bf16): C [SC][np16 + 8] | x [SC][DV + 8] | state, two terms [2][np16][DV + 8], before them B [SC][np16 + 8] in the same place
static size_t ssm_out_smem(int np, int DV) {
    const size_t state = (size_t)2 * up16(np) * (DV + 8), b = (size_t)SC * (up16(np) + 8);
    return ((size_t)SC * (up16(np) + 8) + (size_t)SC * (DV + 8) + (state > b ? state : b)) * 2;
}

template <int DV>
__global__ void __launch_bounds__(128)
skn_ssm_out_kernel(skn_ssm_args a, int T, int nchunks, int per) {
    extern __shared__ __align__(16) uint8_t smb[];
    __shared__ float cum_s[SC], dt_s[SC];
    skn_pdl_launch_dependents();
    skn_pdl_wait();
    const int np16 = up16(a.np), bs = np16 + 8, xs = DV + 8;
    __nv_bfloat16 *C = reinterpret_cast<__nv_bfloat16 *>(smb), *X = C + SC * bs, *St = X + SC * xs, *B = St;
    const int c = blockIdx.x, h0 = blockIdx.y * per, seq = blockIdx.z, t0 = c * SC, L = min(SC, T - t0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int channels = skn_ssm_channels(a.heads, a.vp, a.groups, a.np), inner = a.heads * a.vp, g = h0 / (a.heads / a.groups);
    const int64_t row0 = (int64_t)seq * T + t0;
    const __nv_bfloat16 *rows = a.xbc + row0 * channels;
    ssm_load_rows(B, bs, rows + inner + g * a.np, channels, L, a.np, np16);
    ssm_load_rows(C, bs, rows + inner + (a.groups + g) * a.np, channels, L, a.np, np16);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // C . B of the warp's 16 tokens, shared by the CTA's heads
    const int m0 = warp * 16, gr = lane >> 2, gc = (lane & 3) * 2;
    float s[SC / 8][4];
#pragma unroll
    for (int i = 0; i < SC / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    for (int kk = 0; kk < np16; kk += 16) {
        uint32_t af[4];
        ldsm4(af, skn_smem_u32(C + (size_t)(m0 + (lane & 15)) * bs + kk + (lane >> 4) * 8));
#pragma unroll
        for (int n = 0; n < SC / 16; ++n) {
            if (n > warp) continue;                 // later tokens
            uint32_t bf[4];
            ldsm4(bf, skn_smem_u32(B + (size_t)(n * 16 + (lane & 7) + ((lane >> 4) << 3)) * bs + kk + ((lane >> 3) & 1) * 8));
            mma_bf16(s[2 * n], af, bf[0], bf[1]);
            mma_bf16(s[2 * n + 1], af, bf[2], bf[3]);
        }
    }
    for (int h = h0; h < h0 + per; ++h) {
        __syncthreads();                            // the head before is done with x, the state and the decays
        ssm_load_tile<DV>(X, rows + h * a.vp, channels, SC, L, a.vp);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (tid < SC) {
            const int64_t at = (row0 + min(tid, L - 1)) * a.heads + h;
            cum_s[tid] = a.cum[at];
            dt_s[tid] = tid < L ? a.dt[at] : 0.f;
        }
        const __nv_bfloat16 *S = a.starts + (((int64_t)seq * nchunks + c) * a.heads + h) * 2 * a.np * a.vp;
#pragma unroll
        for (int x = 0; x < 2; ++x) ssm_load_tile<DV>(St + (size_t)x * np16 * xs, S + (int64_t)x * a.np * a.vp, a.vp, np16, a.np, a.vp);
        asm volatile("cp.async.commit_group;" ::: "memory");
        // on their way into L2: this head's gate rows, the next one's state and x
        for (int c = 0; c < a.vp; c += 32)
            if (tid < L) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.proj + (row0 + tid) * a.ld + h * a.vp + c));
        if (h + 1 < h0 + per) {
            const __nv_bfloat16 *next = S + (int64_t)2 * a.np * a.vp;
            for (int i = tid * 64; i < 2 * a.np * a.vp; i += 128 * 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(next + i));
            if (tid < L) asm volatile("prefetch.global.L2 [%0];" ::"l"(rows + (int64_t)tid * channels + (h + 1) * a.vp));
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        float o[DV / 8][4];
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
        for (int kk = 0; kk < np16; kk += 16) {
            uint32_t af[4];
            ldsm4(af, skn_smem_u32(C + (size_t)(m0 + (lane & 15)) * bs + kk + (lane >> 4) * 8));
#pragma unroll
            for (int x = 1; x >= 0; --x)
#pragma unroll
                for (int n = 0; n < DV / 16; ++n) {
                    uint32_t bf[4];
                    ldsm4t(bf, skn_smem_u32(St + ((size_t)x * np16 + kk + (lane & 7) + ((lane >> 3) & 1) * 8) * xs + n * 16 + (lane >> 4) * 8));
                    mma_bf16(o[2 * n], af, bf[0], bf[1]);
                    mma_bf16(o[2 * n + 1], af, bf[2], bf[3]);
                }
        }
        const float ci[2] = {cum_s[m0 + gr], cum_s[m0 + gr + 8]}, ei[2] = {__expf(ci[0]), __expf(ci[1])};
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) {
            o[i][0] *= ei[0]; o[i][1] *= ei[0];
            o[i][2] *= ei[1]; o[i][3] *= ei[1];
        }
#pragma unroll
        for (int kk = 0; kk < SC / 16; ++kk) {
            if (kk > warp) continue;
            uint32_t pf[2][4];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int nt = 2 * kk + (x >> 1), r = x & 1, i = m0 + gr + r * 8, j = nt * 8 + gc;
                const float p0 = j <= i ? s[nt][r * 2] * __expf(ci[r] - cum_s[j]) * dt_s[j] : 0.f;
                const float p1 = j + 1 <= i ? s[nt][r * 2 + 1] * __expf(ci[r] - cum_s[j + 1]) * dt_s[j + 1] : 0.f;
                uint32_t t2[2];
                bf16_terms<2>(p0, p1, t2);
                pf[0][x] = t2[0];
                pf[1][x] = t2[1];
            }
#pragma unroll
            for (int n = 0; n < DV / 16; ++n) {
                uint32_t bf[4];
                ldsm4t(bf, skn_smem_u32(X + (size_t)(kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * xs + n * 16 + (lane >> 4) * 8));
#pragma unroll
                for (int y = 1; y >= 0; --y) {
                    mma_bf16(o[2 * n], pf[y], bf[0], bf[1]);
                    mma_bf16(o[2 * n + 1], pf[y], bf[2], bf[3]);
                }
            }
        }
        const float dv = a.d[h];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int i = m0 + gr + r * 8;
            if (i >= L) continue;
            const int64_t m = row0 + i;
            const float *zr = a.proj + m * a.ld + h * a.vp;
            float *yr = a.y + m * a.ld_y + h * a.vp;
            float2 z[DV / 8];                       // loaded before the first store
#pragma unroll
            for (int n = 0; n < DV / 8; ++n) z[n] = n * 8 + gc < a.vp ? __ldcg(reinterpret_cast<const float2 *>(zr + n * 8 + gc)) : make_float2(0.f, 0.f);
#pragma unroll
            for (int n = 0; n < DV / 8; ++n) {
                const int v = n * 8 + gc;
                if (v >= a.vp) continue;
                const uint32_t xw = *reinterpret_cast<const uint32_t *>(X + i * xs + v);
                float2 y;
                y.x = fmaf(dv, __uint_as_float(xw << 16), o[n][r * 2]) * ssm_silu_fast(z[n].x);
                y.y = fmaf(dv, __uint_as_float(xw & 0xFFFF0000u), o[n][r * 2 + 1]) * ssm_silu_fast(z[n].y);
                *reinterpret_cast<float2 *>(yr + v) = y;
            }
        }
    }
}

bool skn_ssm_chunks_fit(int vp, int np) { return vp <= 128 && np <= 256 && ssm_out_smem(np, vp <= 32 ? 32 : vp <= 64 ? 64 : 128) <= 200 * 1024; }

template <int DV>
static cudaError_t launch_chunks(const skn_step &s, const skn_ssm_args &a, cudaStream_t st) {
    const int nchunks = (s.T + SC - 1) / SC, channels = skn_ssm_channels(a.heads, a.vp, a.groups, a.np);
    const int ctiles = (channels / 4 + 127) / 128, htiles = (a.heads + 31) / 32;
    const dim3 vgrid(ctiles + htiles, (s.T + CV_TOKENS - 1) / CV_TOKENS, s.n_seqs);
    cudaError_t e = a.taps == 4   ? skn_launch_pdl(skn_ssm_conv_kernel<4>, vgrid, dim3(128), 0, st, 1, a, s, (const float *)a.ring->d, a.ring->v_pitch, ctiles)
                    : a.taps == 2 ? skn_launch_pdl(skn_ssm_conv_kernel<2>, vgrid, dim3(128), 0, st, 1, a, s, (const float *)a.ring->d, a.ring->v_pitch, ctiles)
                    : a.taps == 3 ? skn_launch_pdl(skn_ssm_conv_kernel<3>, vgrid, dim3(128), 0, st, 1, a, s, (const float *)a.ring->d, a.ring->v_pitch, ctiles)
                                  : skn_launch_pdl(skn_ssm_conv_kernel<0>, vgrid, dim3(128), 0, st, 1, a, s, (const float *)a.ring->d, a.ring->v_pitch, ctiles);
    if (e != cudaSuccess) return e;
    // heads of a CTA: as many as share B and C, while the grid still fills the GPU
    const int group = a.heads / a.groups;
    int per = 1;
    for (int p = 2; p <= 8; p *= 2)
        if (group % p == 0 && (int64_t)nchunks * s.n_seqs * (a.heads / p) >= 1024) per = p;
    const dim3 grid(nchunks, a.heads / per, s.n_seqs);
    if ((e = cudaFuncSetAttribute(skn_ssm_chunk_kernel<DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)) != cudaSuccess) return e;
    if ((e = skn_launch_pdl(skn_ssm_chunk_kernel<DV>, grid, dim3(128), ssm_chunk_smem(a.np, DV), st, 1, a, s.T, nchunks, per)) != cudaSuccess) return e;
    const int64_t elems = (int64_t)a.heads * a.np * (a.vp / 4);
    const int blocks = (int)((elems + 127) / 128), file = (int)(((int64_t)(a.taps - 1) * channels + 127) / 128);
    e = skn_launch_pdl(skn_ssm_scan_kernel, dim3(blocks + file, s.n_seqs), dim3(128), 0, st, 1, a, s, a.state->d, a.ring->d, a.ring->v_pitch, nchunks, blocks);
    if (e != cudaSuccess) return e;
    if ((e = cudaFuncSetAttribute(skn_ssm_out_kernel<DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)) != cudaSuccess) return e;
    return skn_launch_pdl(skn_ssm_out_kernel<DV>, grid, dim3(128), ssm_out_smem(a.np, DV), st, 1, a, s.T, nchunks, per);
}

cudaError_t skn_launch_ssm_chunks(const skn_step &s, const skn_ssm_args &a, cudaStream_t st) {
    return a.vp <= 32 ? launch_chunks<32>(s, a, st) : a.vp <= 64 ? launch_chunks<64>(s, a, st) : launch_chunks<128>(s, a, st);
}

int32_t skn_check_ssm_spec(skn_ctx *ctx, const skn_ssm_spec *s) {
    if (s->heads < 1 || s->vdim < 1 || s->state < 1 || s->groups < 1 || s->taps < 1 || s->norm_groups < 1) return skn_fail(ctx, SKN_ERR_ARG, "invalid state space geometry");
    if (s->heads % s->groups || (s->heads * s->vdim) % s->norm_groups || s->state > SKN_ATTN_MAX_DIM || s->vdim > SKN_ATTN_MAX_DIM)
        return skn_fail(ctx, SKN_ERR_SHAPE, "Shapes do not align.");
    return SKN_OK;
}
