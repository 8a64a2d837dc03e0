// Generalized delta rule of the block engine (k2t_block_kernels.h), fp32 throughout: per head a state S [key][value] with
//   S_t = diag(w) S_(t-1) - (a u)(u^T S_(t-1)) + k v^T,   o_t = S_t^T r,
// w the decay and a the removal rate per key channel, u the unit key.  Columns of S do not meet, so a column group of a head is
// an independent chain.
//   * delta_step_kernel (one token): CTA = head.  The state is requested before the dependency wait (only the same layer's
//     previous step wrote it), then coefficients, recurrence, per-head norm, output gate and the activation of the output
//     projection in one launch.
//   * prompts: delta_prep_kernel writes the coefficients of every (head, token) as one record, delta_scan_kernel walks the
//     tokens - CTA = 16 columns of a head, warp = 4 columns, eight lanes share a column's keys - with the records streamed
//     through a ring of bulk copies and packed fp32 pairs (fma.rn.f32x2), delta_post_kernel norms and gates.
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
__device__ __forceinline__ ulonglong2 lds2(uint32_t saddr) {
    ulonglong2 v;
    asm volatile("ld.shared.v2.u64 {%0, %1}, [%2];" : "=l"(v.x), "=l"(v.y) : "r"(saddr));
    return v;
}

// ------------------------------------------------------------------------------------------------ one token
// thread = (four columns, sixteen keys): drow^2 / 64 threads
constexpr uint32_t ST_KEYS = 16;
inline uint32_t step_threads(uint32_t drow) { return std::max(64u, drow / 4 * (drow / ST_KEYS)); }
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

// one warp per (token, head): record [w - 1 | a u | u | k | r | v], drow floats each
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaArgs a, uint32_t n_tok) {
    const uint32_t lane = threadIdx.x & 31, h = blockIdx.y, t = blockIdx.x * 8 + (threadIdx.x >> 5), D = a.drow, dim = a.dim, HD = a.heads * dim;
    pdl_wait();
    pdl_trigger();
    if (t >= n_tok) return;
    const float *in = a.in + t * a.in_stride + h * dim, *lg = a.decay_logit + t * a.logit_stride + h * dim;
    float *rec = a.rec + ((size_t)h * n_tok + t) * 6 * D;
    float kk = 0.0f;
    for (uint32_t i = lane; i < dim; i += 32) { const float k = __ldcg(in + HD + i); kk = __fmaf_rn(k, k, kk); }
    const float inv_k = 1.0f / sqrtf(warp_sum(kk) + a.unit_eps);
    for (uint32_t i = lane; i < D; i += 32) {
        float w = 0.0f, au = 0.0f, u = 0.0f, k = 0.0f, r = 0.0f, v = 0.0f;
        if (i < dim) {
            k = __ldcg(in + HD + i);
            u = k * inv_k;
            w = decay_minus_one(a.decay_scale, __ldcg(lg + i) + __ldg(a.decay_bias + h * dim + i));
            au = sigmoidf(__ldcg(in + 4 * HD + i) + __ldg(a.rate_bias + h * dim + i)) * u;
            r = __ldcg(in + i);
            v = __ldcg(in + 2 * HD + i);
        }
        rec[i] = w; rec[D + i] = au; rec[2 * D + i] = u; rec[3 * D + i] = k; rec[4 * D + i] = r; rec[5 * D + i] = v;
    }
}

constexpr uint32_t SC_STAGES = 3, SC_FLOATS = 6144;        // ring: stages of SC_FLOATS floats (1024 / drow records)
constexpr uint32_t SC_WAIT_LIMIT = 1u << 22;

template <int KI>       // drow = 32 KI: lane kl of a column's eight holds keys 4 (8 i + kl) .. + 3, i < KI
__global__ void __launch_bounds__(128) delta_scan_kernel(const float *__restrict__ rec, uint32_t n_tok, float *__restrict__ state, float *__restrict__ o, uint32_t heads,
                                                        uint32_t *__restrict__ err_flag) {
    extern __shared__ __align__(128) float ring[];
    __shared__ __align__(8) uint64_t bars[SC_STAGES];
    constexpr uint32_t D = 32 * KI, TB = 1024 / D, REC = 6 * D;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, kl = lane & 7u, col = blockIdx.x * 16 + warp * 4 + (lane >> 3);
    const uint32_t bar = (uint32_t)__cvta_generic_to_shared(bars), rb = (uint32_t)__cvta_generic_to_shared(ring);
    const float *src = rec + (size_t)h * n_tok * REC;
    const uint32_t chunks = (n_tok + TB - 1) / TB;
    if (tid == 0) {
        for (uint32_t i = 0; i < SC_STAGES; ++i) mbar_init(bar + 8 * i, 1);
        fence_mbar_init();
    }
    float *sp = state + (size_t)h * D * D + col;
    uint64_t s[KI][2];
#pragma unroll
    for (int i = 0; i < KI; ++i) {
        const uint32_t key = (i * 8 + kl) * 4;
        s[i][0] = pk(__ldcg(sp + (size_t)key * D), __ldcg(sp + (size_t)(key + 1) * D));
        s[i][1] = pk(__ldcg(sp + (size_t)(key + 2) * D), __ldcg(sp + (size_t)(key + 3) * D));
    }
    pdl_wait();
    pdl_trigger();
    __syncthreads();
    auto request = [&](uint32_t c) {
        const uint32_t n = min(TB, n_tok - c * TB);
        mbar_expect_tx(bar + 8 * (c % SC_STAGES), n * REC * 4);
        bulk_g2s(rb + (c % SC_STAGES) * SC_FLOATS * 4, src + (size_t)c * TB * REC, n * REC * 4, bar + 8 * (c % SC_STAGES));
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
        const uint32_t n = min(TB, n_tok - c * TB);
        uint32_t at = rb + (c % SC_STAGES) * SC_FLOATS * 4;
#pragma unroll 2
        for (uint32_t t = 0; t < n; ++t, at += REC * 4) {
            const uint32_t ak = at + kl * 16;
            uint64_t d0 = 0, d1 = 0;
#pragma unroll
            for (int i = 0; i < KI; ++i) {
                const ulonglong2 u = lds2(ak + 2 * D * 4 + i * 128);
                d0 = fma2(u.x, s[i][0], d0);
                d1 = fma2(u.y, s[i][1], d1);
            }
            float v;
            asm volatile("ld.shared.f32 %0, [%1];" : "=f"(v) : "r"(at + (5 * D + col) * 4));
            const uint64_t v2 = pk(v, v);
#pragma unroll
            for (int i = 0; i < KI; ++i) {          // w S + k v^T does not need the reduced product
                const ulonglong2 w = lds2(ak + i * 128), k = lds2(ak + 3 * D * 4 + i * 128);
                s[i][0] = fma2(w.x, s[i][0], fma2(k.x, v2, s[i][0]));
                s[i][1] = fma2(w.y, s[i][1], fma2(k.y, v2, s[i][1]));
            }
            float e0, e1, e2, e3;
            upk(d0, e0, e1);
            upk(d1, e2, e3);
            float cc = __fadd_rn(__fadd_rn(e0, e1), __fadd_rn(e2, e3));
            cc = __fadd_rn(cc, __shfl_xor_sync(0xffffffffu, cc, 1));
            cc = __fadd_rn(cc, __shfl_xor_sync(0xffffffffu, cc, 2));
            cc = __fadd_rn(cc, __shfl_xor_sync(0xffffffffu, cc, 4));
            const uint64_t c2 = pk(-cc, -cc);
            uint64_t o0 = 0, o1 = 0;
#pragma unroll
            for (int i = 0; i < KI; ++i) {
                const ulonglong2 au = lds2(ak + D * 4 + i * 128), r = lds2(ak + 4 * D * 4 + i * 128);
                s[i][0] = fma2(au.x, c2, s[i][0]);
                s[i][1] = fma2(au.y, c2, s[i][1]);
                o0 = fma2(r.x, s[i][0], o0);
                o1 = fma2(r.y, s[i][1], o1);
            }
            upk(o0, e0, e1);
            upk(o1, e2, e3);
            float oo = __fadd_rn(__fadd_rn(e0, e1), __fadd_rn(e2, e3));
            oo = __fadd_rn(oo, __shfl_xor_sync(0xffffffffu, oo, 1));
            oo = __fadd_rn(oo, __shfl_xor_sync(0xffffffffu, oo, 2));
            oo = __fadd_rn(oo, __shfl_xor_sync(0xffffffffu, oo, 4));
            if (kl == 0) o[((size_t)(c * TB + t) * heads + h) * D + col] = oo;
        }
        __syncthreads();                        // the stage is free
        if (tid == 0 && c + SC_STAGES < chunks) request(c + SC_STAGES);
    }
#pragma unroll
    for (int i = 0; i < KI; ++i) {
        const uint32_t key = (i * 8 + kl) * 4;
        float e0, e1, e2, e3;
        upk(s[i][0], e0, e1);
        upk(s[i][1], e2, e3);
        sp[(size_t)key * D] = e0; sp[(size_t)(key + 1) * D] = e1; sp[(size_t)(key + 2) * D] = e2; sp[(size_t)(key + 3) * D] = e3;
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

template <int KI> cudaError_t scan_ki(cudaStream_t s, const DeltaArgs &a, uint32_t n_tok, bool pdl) {
    const size_t smem = SC_STAGES * SC_FLOATS * 4;
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(delta_scan_kernel<KI>), smem);
    if (e != cudaSuccess) return e;
    return launch_kernel(delta_scan_kernel<KI>, dim3(2 * KI, a.heads), dim3(128), smem, s, pdl, a.rec, n_tok, a.state, a.o, a.heads, a.err_flag);
}

}  // namespace

uint32_t delta_row(uint32_t dim) { return dim <= 256 ? (dim + 31u) & ~31u : 0u; }
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
    cudaError_t e = launch_kernel(delta_prep_kernel, grid, dim3(256), 0, s, pdl, a, n_tok);
    if (e != cudaSuccess) return e;
    switch (a.drow / 32) {
        case 1: e = scan_ki<1>(s, a, n_tok, pdl); break;
        case 2: e = scan_ki<2>(s, a, n_tok, pdl); break;
        case 3: e = scan_ki<3>(s, a, n_tok, pdl); break;
        case 4: e = scan_ki<4>(s, a, n_tok, pdl); break;
        case 5: e = scan_ki<5>(s, a, n_tok, pdl); break;
        case 6: e = scan_ki<6>(s, a, n_tok, pdl); break;
        case 7: e = scan_ki<7>(s, a, n_tok, pdl); break;
        case 8: e = scan_ki<8>(s, a, n_tok, pdl); break;
        default: e = cudaErrorInvalidValue;
    }
    if (e != cudaSuccess) return e;
    return launch_kernel(f32 ? delta_post_kernel<true> : delta_post_kernel<false>, grid, dim3(256), 0, s, pdl, a, n_tok);
}

}  // namespace k2t
