// Generalized delta rule of the block engine (k2t_block_kernels.h), fp32 throughout: per head a state S [key][value] with
//   S_t = diag(w) S_(t-1) - (a u)(u^T S_(t-1)) + k v^T,   o_t = S_t^T r,
// w the decay and a the removal rate per key channel, u the unit key.  Columns of S do not meet, so a column group of a head is
// an independent chain.
//   * delta_step_kernel (one token): CTA = head.  The state is requested before the dependency wait (only the same layer's
//     previous step wrote it), then coefficients, recurrence, per-head norm, output gate and the activation of the output
//     projection in one launch.
//   * prompts: delta_prep_kernel writes the coefficients of every head and group of four tokens as one record,
//     delta_scan_kernel walks the groups - a warp holds four columns, its lanes share the keys - with the records streamed through
//     a ring of bulk copies and packed fp32 pairs (fma.rn.f32x2), delta_post_kernel norms and gates.
#include <algorithm>

#include "k2t_block_kernels.h"
#include "k2t_dense.cuh"

namespace k2t {
namespace {

__device__ __forceinline__ float sigmoidf(float x) { return 1.0f / (1.0f + expf(-x)); }
// Decays are kept as w - 1: a channel that decays by a hair per token would lose that hair in the rounding of w, the same way
// at every token, and a state carried over thousands of tokens would show it.
__device__ __forceinline__ float decay_minus_one(float scale, float logit) { return expm1f(-scale * sigmoidf(logit)); }

// ---- packed fp32 pairs
__device__ __forceinline__ uint64_t pk(float a, float b) { uint64_t r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b)); return r; }
__device__ __forceinline__ void upk(uint64_t v, float &a, float &b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) { uint64_t r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }

// ------------------------------------------------------------------------------------------------ one token
// thread = (four columns, sixteen keys): drow^2 / 64 threads
constexpr uint32_t ST_KEYS = 16;
inline uint32_t step_threads(uint32_t drow) { return std::max(128u, drow / 4 * (drow / ST_KEYS)); }
inline size_t step_smem(uint32_t drow, uint32_t rank_pad) { return ((size_t)drow * (6 + drow / ST_KEYS) + rank_pad) * 4; }

template <bool F32>
__global__ void __launch_bounds__(256) delta_step_kernel(const DeltaArgs a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32];
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, D = a.drow, dim = a.dim, nthr = blockDim.x;
    const uint32_t quads = D / 4, slices = D / ST_KEYS, q = tid % quads, sl = tid / quads, rank_pad = (a.rank + 63) / 64 * 64;
    const bool live = sl < slices;
    float *s_w = sm, *s_au = s_w + D, *s_u = s_au + D, *s_k = s_u + D, *s_r = s_k + D, *s_v = s_r + D, *s_red = s_v + D, *s_t = s_red + slices * D;
    float4 st[ST_KEYS];
    float *state = a.state + (size_t)h * D * D + (size_t)(sl * ST_KEYS) * D + q * 4;
    if (live)
#pragma unroll
        for (uint32_t i = 0; i < ST_KEYS; ++i) st[i] = __ldcg(reinterpret_cast<const float4 *>(state + (size_t)i * D));
    for (uint32_t i = tid; i < 6 * D; i += nthr) sm[i] = 0.0f;
    for (uint32_t i = tid; i < rank_pad; i += nthr) s_t[i] = 0.0f;
    if (!F32)           // the head's rows of the decay product: weights, fetched while the predecessor runs
        for (uint32_t i = tid; i < dim * a.decay.panels; i += nthr)
            asm volatile("prefetch.global.L2 [%0];" ::"l"(static_cast<const char *>(a.decay.base) + ((size_t)(i / dim) * a.decay.rows_pad + h * dim + i % dim) * 128));
    pdl_wait();
    pdl_trigger();
    __syncthreads();
    const uint32_t HD = a.heads * dim;
    const float *in = a.in + h * dim;
    float kk[1] = {0.0f};
    for (uint32_t i = tid; i < dim; i += nthr) {
        const float k = __ldcg(in + HD + i);
        s_r[i] = __ldcg(in + i);
        s_k[i] = k;
        s_v[i] = __ldcg(in + 2 * HD + i);
        kk[0] = __fmaf_rn(k, k, kk[0]);
    }
    for (uint32_t i = tid; i < a.rank; i += nthr) s_t[i] = tanhf(__ldcg(a.in + 5 * HD + i));
    block_sum<1>(kk, scratch);                          // its barriers also publish s_t, s_k
    const float inv_k = 1.0f / sqrtf(kk[0] + a.unit_eps);
    const uint32_t sub = lane & 7u;
#pragma unroll 4
    for (uint32_t r0 = warp * 4; r0 < dim; r0 += nthr / 8) {
        const uint32_t i = r0 + (lane >> 3), ii = min(i, dim - 1), c = h * dim + ii;
        const float z = row_dot8<F32>(a.decay, c, 0, a.decay.panels, s_t, sub) + __ldg(a.decay_bias + c);
        if (i < dim && sub == 0) {
            const float u = s_k[i] * inv_k;
            s_w[i] = decay_minus_one(a.decay_scale, z);
            s_u[i] = u;
            s_au[i] = sigmoidf(__ldcg(in + 4 * HD + i) + __ldg(a.rate_bias + c)) * u;
        }
    }
    __syncthreads();
    if (live) {
        float4 c = make_float4(0, 0, 0, 0);
#pragma unroll
        for (uint32_t i = 0; i < ST_KEYS; ++i) {
            const float u = s_u[sl * ST_KEYS + i];
            c.x = __fmaf_rn(u, st[i].x, c.x); c.y = __fmaf_rn(u, st[i].y, c.y); c.z = __fmaf_rn(u, st[i].z, c.z); c.w = __fmaf_rn(u, st[i].w, c.w);
        }
        *reinterpret_cast<float4 *>(s_red + sl * D + q * 4) = c;
    }
    __syncthreads();
    float4 o = make_float4(0, 0, 0, 0);
    if (live) {
        float4 c = make_float4(0, 0, 0, 0);
        for (uint32_t s = 0; s < slices; ++s) {
            const float4 p = *reinterpret_cast<const float4 *>(s_red + s * D + q * 4);
            c.x += p.x; c.y += p.y; c.z += p.z; c.w += p.w;
        }
        const float4 v = *reinterpret_cast<const float4 *>(s_v + q * 4);
#pragma unroll
        for (uint32_t i = 0; i < ST_KEYS; ++i) {
            const uint32_t key = sl * ST_KEYS + i;
            const float w = s_w[key], au = -s_au[key], k = s_k[key], r = s_r[key];
            st[i].x = __fmaf_rn(au, c.x, __fmaf_rn(w, st[i].x, __fmaf_rn(k, v.x, st[i].x))); st[i].y = __fmaf_rn(au, c.y, __fmaf_rn(w, st[i].y, __fmaf_rn(k, v.y, st[i].y)));
            st[i].z = __fmaf_rn(au, c.z, __fmaf_rn(w, st[i].z, __fmaf_rn(k, v.z, st[i].z))); st[i].w = __fmaf_rn(au, c.w, __fmaf_rn(w, st[i].w, __fmaf_rn(k, v.w, st[i].w)));
            o.x = __fmaf_rn(r, st[i].x, o.x); o.y = __fmaf_rn(r, st[i].y, o.y); o.z = __fmaf_rn(r, st[i].z, o.z); o.w = __fmaf_rn(r, st[i].w, o.w);
            *reinterpret_cast<float4 *>(state + (size_t)i * D) = st[i];
        }
    }
    __syncthreads();                                    // every slice has read the partial sums
    if (live) *reinterpret_cast<float4 *>(s_red + sl * D + q * 4) = o;
    __syncthreads();
    float so[1] = {0.0f};
    for (uint32_t j = tid; j < dim; j += nthr) {
        float v = 0.0f;
        for (uint32_t s = 0; s < slices; ++s) v += s_red[s * D + j];
        s_v[j] = v;
        so[0] = __fmaf_rn(v, v, so[0]);
    }
    block_sum<1>(so, scratch);
    const float inv = 1.0f / sqrtf(so[0] / (float)dim + a.eps);
    for (uint32_t j = tid; j < dim; j += nthr)
        act_store<F32>(a.out, 0, h * dim + j, s_v[j] * inv * __ldg(a.norm + h * dim + j) * sigmoidf(__ldcg(in + 3 * HD + j)));
}

// ------------------------------------------------------------------------------------------------ prompts
template <bool F32>
__global__ void __launch_bounds__(256) delta_tanh_kernel(const float *__restrict__ in, size_t in_stride, uint32_t rank, uint32_t n_tok, const Act out) {
    const uint32_t i = blockIdx.x * 256 + threadIdx.x;
    pdl_wait();
    pdl_trigger();
    if (i >= n_tok * rank) return;
    act_store<F32>(out, i / rank, i % rank, tanhf(__ldcg(in + (i / rank) * in_stride + i % rank)));
}

// Prompts run in groups of four tokens.  With S the state ahead of a group, the products c_t = u_t^T S_(t-1) the removals need are
//   c_t = U_t^T S + sum over s < t of (G_ts v_s - H_ts c_s),   U_t = u_t w_0 .. w_(t-1),
//   G_ts = (u_t w_(s+1) .. w_(t-1))^T k_s,   H_ts = (u_t w_(s+1) .. w_(t-1))^T (a u)_s   (products by key channel),
// so the four reductions over the keys of a column go side by side and one round of shuffles serves four tokens.  A group's
// record: four times [w - 1 | a u | U | k | r | v] of drow floats, then G and H of the pairs (1,0) (2,0) (2,1) (3,0) (3,1) (3,2).
constexpr uint32_t GROUP = 4;
__host__ __device__ constexpr uint32_t group_floats(uint32_t drow) { return GROUP * 6 * drow + 16; }

template <int NI>       // drow = 32 NI; one warp per (group, head)
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaArgs a, uint32_t n_tok) {
    constexpr uint32_t D = 32 * NI;
    const uint32_t lane = threadIdx.x & 31, h = blockIdx.y, g = blockIdx.x * 8 + (threadIdx.x >> 5), dim = a.dim, HD = a.heads * dim, groups = (n_tok + GROUP - 1) / GROUP;
    pdl_wait();
    pdl_trigger();
    if (g >= groups) return;
    float *rec = a.rec + ((size_t)h * groups + g) * group_floats(D);
    float k[GROUP][NI], inv_k[GROUP], sums[12];
#pragma unroll
    for (uint32_t t = 0; t < GROUP; ++t) {
        const uint32_t tok = g * GROUP + t;
        const float *in = a.in + tok * a.in_stride + h * dim;
        float kk = 0.0f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const uint32_t c = lane + 32 * i;
            k[t][i] = tok < n_tok && c < dim ? __ldcg(in + HD + c) : 0.0f;
            kk = __fmaf_rn(k[t][i], k[t][i], kk);
        }
        inv_k[t] = 1.0f / sqrtf(warp_sum(kk) + a.unit_eps);
    }
#pragma unroll
    for (int j = 0; j < 12; ++j) sums[j] = 0.0f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const uint32_t c = lane + 32 * i;
        float w[GROUP], au[GROUP];
#pragma unroll
        for (uint32_t t = 0; t < GROUP; ++t) {
            const uint32_t tok = g * GROUP + t;
            const float *in = a.in + tok * a.in_stride + h * dim;
            float d = 0.0f, r = 0.0f, v = 0.0f;
            au[t] = 0.0f;
            float u = k[t][i] * inv_k[t];
            if (tok < n_tok && c < dim) {
                d = decay_minus_one(a.decay_scale, __ldcg(a.decay_logit + tok * a.logit_stride + h * dim + c) + __ldg(a.decay_bias + h * dim + c));
                au[t] = sigmoidf(__ldcg(in + 4 * HD + c) + __ldg(a.rate_bias + h * dim + c)) * u;
                r = __ldcg(in + c);
                v = __ldcg(in + 2 * HD + c);
            }
            w[t] = 1.0f + d;
            // u w_(t-1) .. w_(s+1) against k_s and (a u)_s, s from t - 1 down
#pragma unroll
            for (int s = GROUP - 2; s >= 0; --s)
                if (s < (int)t) {
                    const int pair = (int)t * ((int)t - 1) / 2 + s;
                    sums[pair] = __fmaf_rn(u, k[s][i], sums[pair]);
                    sums[6 + pair] = __fmaf_rn(u, au[s], sums[6 + pair]);
                    u *= w[s];
                }
            float *q = rec + t * 6 * D + c;
            q[0] = d; q[D] = au[t]; q[2 * D] = u; q[3 * D] = k[t][i]; q[4 * D] = r; q[5 * D] = v;
        }
    }
    float mine = 0.0f;
#pragma unroll
    for (int j = 0; j < 12; ++j) {
        const float v = warp_sum(sums[j]);
        if ((int)lane == j) mine = v;
    }
    if (lane < 16) rec[GROUP * 6 * D + lane] = mine;
}

constexpr uint32_t SC_STAGES = 3, SC_COLS = 4;
constexpr uint32_t SC_WAIT_LIMIT = 1u << 22;
__host__ __device__ constexpr uint32_t stage_groups(uint32_t drow) { return drow >= 256 ? 1u : 256u / drow; }

// Sixteen values per lane summed over the warp: lane l returns the sum of value l / 2 (the exchange halves the values per step).
__device__ __forceinline__ float warp_sum16(float (&v)[16], uint32_t lane) {
#pragma unroll
    for (int w = 8; w > 0; w >>= 1)
#pragma unroll
        for (int i = 0; i < w; ++i) {
            const bool up = (lane & (2 * w)) != 0;
            const float give = up ? v[i] : v[i + w], keep = up ? v[i + w] : v[i];
            v[i] = __fadd_rn(keep, __shfl_xor_sync(0xffffffffu, give, 2 * w));
        }
    return __fadd_rn(v[0], __shfl_xor_sync(0xffffffffu, v[0], 1));
}

// CTA = four warps, warp = four columns of a head; the 32 lanes share the keys: lane l holds the key pairs 2 (32 i + l), i < KP
// (drow = 64 KP), so a record vector is read once per warp, 256 consecutive bytes per load.
template <int KP>
__global__ void __launch_bounds__(128) delta_scan_kernel(const float *__restrict__ rec, uint32_t n_tok, float *__restrict__ state, float *__restrict__ o, uint32_t heads,
                                                        uint32_t *__restrict__ err_flag) {
    extern __shared__ __align__(128) float ring[];
    __shared__ __align__(8) uint64_t bars[SC_STAGES];
    constexpr uint32_t D = 64 * KP, GF = group_floats(D), SG = stage_groups(D), STAGE = SG * GF;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, col = (blockIdx.x * 4 + warp) * SC_COLS;
    const uint32_t bar = (uint32_t)__cvta_generic_to_shared(bars), rb = (uint32_t)__cvta_generic_to_shared(ring);
    const uint32_t groups = (n_tok + GROUP - 1) / GROUP, chunks = (groups + SG - 1) / SG;
    const float *src = rec + (size_t)h * groups * GF;
    if (tid == 0) {
        for (uint32_t i = 0; i < SC_STAGES; ++i) mbar_init(bar + 8 * i, 1);
        fence_mbar_init();
    }
    float *sp = state + (size_t)h * D * D + col;
    uint64_t s[SC_COLS][KP];
#pragma unroll
    for (int i = 0; i < KP; ++i) {
        const float *q = sp + (size_t)((i * 32 + lane) * 2) * D;
        const float4 e = __ldcg(reinterpret_cast<const float4 *>(q)), f = __ldcg(reinterpret_cast<const float4 *>(q + D));
        s[0][i] = pk(e.x, f.x); s[1][i] = pk(e.y, f.y); s[2][i] = pk(e.z, f.z); s[3][i] = pk(e.w, f.w);
    }
    pdl_wait();
    pdl_trigger();
    __syncthreads();
    auto request = [&](uint32_t c) {
        const uint32_t bytes = min(SG, groups - c * SG) * GF * 4;
        mbar_expect_tx(bar + 8 * (c % SC_STAGES), bytes);
        bulk_g2s(rb + (c % SC_STAGES) * STAGE * 4, src + (size_t)c * STAGE, bytes, bar + 8 * (c % SC_STAGES));
    };
    if (tid == 0)
        for (uint32_t c = 0; c < min(SC_STAGES, chunks); ++c) request(c);
    for (uint32_t c = 0; c < chunks; ++c) {
        bool ok = false;
        for (uint32_t spin = 0; spin < SC_WAIT_LIMIT && !ok; ++spin) ok = mbar_try_wait(bar + 8 * (c % SC_STAGES), (c / SC_STAGES) & 1u);
        if (__syncthreads_or(!ok)) {            // a copy did not land: report, let the others in flight land, leave
            if (tid == 0 && err_flag != nullptr) atomicExch(err_flag, 1u);
            for (uint32_t d = c + 1; d < min(c + SC_STAGES, chunks); ++d)
                for (uint32_t spin = 0; spin < SC_WAIT_LIMIT && !mbar_try_wait(bar + 8 * (d % SC_STAGES), (d / SC_STAGES) & 1u); ++spin) {}
            return;
        }
        const uint32_t n = min(SG, groups - c * SG);
        const float *at = ring + (c % SC_STAGES) * STAGE;
#pragma unroll 1
        for (uint32_t gi = 0; gi < n; ++gi, at += GF) {
            const uint64_t *vec = reinterpret_cast<const uint64_t *>(at) + lane;
            auto part = [&](uint32_t t, uint32_t which, int i) { return vec[(t * 6 + which) * (D / 2) + i * 32]; };
            float d[GROUP * SC_COLS], v[GROUP * SC_COLS];
#pragma unroll
            for (uint32_t t = 0; t < GROUP; ++t) {
                uint64_t p[SC_COLS];
#pragma unroll
                for (int i = 0; i < KP; ++i) {
                    const uint64_t u = part(t, 2, i);
#pragma unroll
                    for (int c2 = 0; c2 < (int)SC_COLS; ++c2) p[c2] = fma2(u, s[c2][i], i == 0 ? 0ull : p[c2]);
                }
                const float4 v4 = *reinterpret_cast<const float4 *>(at + (t * 6 + 5) * D + col);
                v[t * 4] = v4.x; v[t * 4 + 1] = v4.y; v[t * 4 + 2] = v4.z; v[t * 4 + 3] = v4.w;
#pragma unroll
                for (int c2 = 0; c2 < (int)SC_COLS; ++c2) { float e0, e1; upk(p[c2], e0, e1); d[t * 4 + c2] = __fadd_rn(e0, e1); }
            }
            const float dm = warp_sum16(d, lane);
#pragma unroll
            for (int i = 0; i < 16; ++i) d[i] = __shfl_sync(0xffffffffu, dm, 2 * i);
            const float *gh = at + GROUP * 6 * D;
#pragma unroll
            for (uint32_t t = 1; t < GROUP; ++t)
#pragma unroll
                for (uint32_t q = 0; q < t; ++q) {
                    const float g = gh[t * (t - 1) / 2 + q], hh = -gh[6 + t * (t - 1) / 2 + q];
#pragma unroll
                    for (int c2 = 0; c2 < (int)SC_COLS; ++c2) d[t * 4 + c2] = __fmaf_rn(hh, d[q * 4 + c2], __fmaf_rn(g, v[q * 4 + c2], d[t * 4 + c2]));
                }
            float oo[GROUP * SC_COLS];
#pragma unroll
            for (uint32_t t = 0; t < GROUP; ++t) {
                uint64_t v2[SC_COLS], c2n[SC_COLS], p[SC_COLS];
#pragma unroll
                for (int c2 = 0; c2 < (int)SC_COLS; ++c2) { v2[c2] = pk(v[t * 4 + c2], v[t * 4 + c2]); c2n[c2] = pk(-d[t * 4 + c2], -d[t * 4 + c2]); }
#pragma unroll
                for (int i = 0; i < KP; ++i) {
                    const uint64_t w = part(t, 0, i), au = part(t, 1, i), k = part(t, 3, i), r = part(t, 4, i);
#pragma unroll
                    for (int c2 = 0; c2 < (int)SC_COLS; ++c2) {
                        s[c2][i] = fma2(au, c2n[c2], fma2(w, s[c2][i], fma2(k, v2[c2], s[c2][i])));
                        p[c2] = fma2(r, s[c2][i], i == 0 ? 0ull : p[c2]);
                    }
                }
#pragma unroll
                for (int c2 = 0; c2 < (int)SC_COLS; ++c2) { float e0, e1; upk(p[c2], e0, e1); oo[t * 4 + c2] = __fadd_rn(e0, e1); }
            }
            const float om = warp_sum16(oo, lane);
            const uint32_t tok = (c * SG + gi) * GROUP + (lane >> 3);
            if ((lane & 1u) == 0 && tok < n_tok) o[((size_t)tok * heads + h) * D + col + ((lane >> 1) & 3u)] = om;
        }
        __syncthreads();                        // the stage is free
        if (tid == 0 && c + SC_STAGES < chunks) request(c + SC_STAGES);
    }
#pragma unroll
    for (int i = 0; i < KP; ++i) {
        float *q = sp + (size_t)((i * 32 + lane) * 2) * D;
        float4 e, f;
        upk(s[0][i], e.x, f.x); upk(s[1][i], e.y, f.y); upk(s[2][i], e.z, f.z); upk(s[3][i], e.w, f.w);
        *reinterpret_cast<float4 *>(q) = e;
        *reinterpret_cast<float4 *>(q + D) = f;
    }
}

template <bool F32>
__global__ void __launch_bounds__(256) delta_post_kernel(const DeltaArgs a, uint32_t n_tok) {
    const uint32_t lane = threadIdx.x & 31, h = blockIdx.y, t = blockIdx.x * 8 + (threadIdx.x >> 5), dim = a.dim;
    pdl_wait();
    pdl_trigger();
    if (t >= n_tok) return;
    const float *o = a.o + ((size_t)t * a.heads + h) * a.drow, *g = a.in + t * a.in_stride + (size_t)3 * a.heads * dim + h * dim;
    float ss = 0.0f;
    for (uint32_t j = lane; j < dim; j += 32) { const float v = __ldcg(o + j); ss = __fmaf_rn(v, v, ss); }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)dim + a.eps);
    for (uint32_t j = lane; j < dim; j += 32) act_store<F32>(a.out, t, h * dim + j, __ldcg(o + j) * inv * __ldg(a.norm + h * dim + j) * sigmoidf(__ldcg(g + j)));
}

template <int KP> cudaError_t scan_kp(cudaStream_t s, const DeltaArgs &a, uint32_t n_tok, bool pdl) {
    const uint32_t groups = (n_tok + GROUP - 1) / GROUP;
    cudaError_t e = launch_kernel(delta_prep_kernel<2 * KP>, dim3((groups + 7) / 8, a.heads), dim3(256), 0, s, pdl, a, n_tok);
    if (e != cudaSuccess) return e;
    constexpr size_t smem = (size_t)SC_STAGES * stage_groups(64 * KP) * group_floats(64 * KP) * 4;
    e = allow_dynamic_smem(reinterpret_cast<const void *>(delta_scan_kernel<KP>), smem);
    if (e != cudaSuccess) return e;
    return launch_kernel(delta_scan_kernel<KP>, dim3(64 * KP / (4 * SC_COLS), a.heads), dim3(128), smem, s, pdl, a.rec, n_tok, a.state, a.o, a.heads, a.err_flag);
}

}  // namespace

uint32_t delta_row(uint32_t dim) { return dim <= 256 ? (dim + 63u) & ~63u : 0u; }
size_t delta_record_floats(uint32_t n_tok, uint32_t heads, uint32_t drow) { return (size_t)((n_tok + GROUP - 1) / GROUP) * heads * group_floats(drow); }
bool delta_step_fits(const DeltaArgs &a) { return a.drow <= 128 && step_smem(a.drow, (a.rank + 63) / 64 * 64) <= 200 * 1024; }

cudaError_t launch_delta_step(cudaStream_t s, bool f32, const DeltaArgs &a, bool pdl) {
    const size_t smem = step_smem(a.drow, (a.rank + 63) / 64 * 64);
    auto k = f32 ? delta_step_kernel<true> : delta_step_kernel<false>;
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(k), smem);
    if (e != cudaSuccess) return e;
    const uint32_t threads = (step_threads(a.drow) + 31u) & ~31u;
    return launch_kernel(k, dim3(a.heads), dim3(threads), smem, s, pdl, a);
}
cudaError_t launch_delta_tanh(cudaStream_t s, bool f32, const DeltaArgs &a, const Act &out, uint32_t n_tok, bool pdl) {
    return launch_kernel(f32 ? delta_tanh_kernel<true> : delta_tanh_kernel<false>, dim3((n_tok * a.rank + 255) / 256), dim3(256), 0, s, pdl,
                         a.in + (size_t)5 * a.heads * a.dim, a.in_stride, a.rank, n_tok, out);
}
cudaError_t launch_delta_prompt(cudaStream_t s, bool f32, const DeltaArgs &a, uint32_t n_tok, bool pdl) {
    const dim3 grid((n_tok + 7) / 8, a.heads);
    cudaError_t e = cudaErrorInvalidValue;
    switch (a.drow / 64) {
        case 1: e = scan_kp<1>(s, a, n_tok, pdl); break;
        case 2: e = scan_kp<2>(s, a, n_tok, pdl); break;
        case 3: e = scan_kp<3>(s, a, n_tok, pdl); break;
        case 4: e = scan_kp<4>(s, a, n_tok, pdl); break;
        default: break;
    }
    if (e != cudaSuccess) return e;
    return launch_kernel(f32 ? delta_post_kernel<true> : delta_post_kernel<false>, grid, dim3(256), 0, s, pdl, a, n_tok);
}

}  // namespace k2t
