// Embedding, norms, per-layer token input and the polynomial activation of the block engine (k2t_block_kernels.h).
#include <algorithm>

#include "k2t_block_kernels.h"
#include "k2t_dense.cuh"

namespace k2t {
namespace {

// four consecutive values, zeros at and beyond n (k a multiple of 4; rows are padded, so the load itself stays inside)
__device__ __forceinline__ float4 load4(const float *p, uint32_t k, uint32_t n) {
    float4 v = __ldcg(reinterpret_cast<const float4 *>(p + k));
    if (k + 4 > n) {
        if (k + 1 > n) v.x = 0.0f;
        if (k + 2 > n) v.y = 0.0f;
        if (k + 3 > n) v.z = 0.0f;
        v.w = 0.0f;
    }
    return v;
}
__device__ __forceinline__ float sq4(const float4 &v, float acc) {
    return __fmaf_rn(v.x, v.x, __fmaf_rn(v.y, v.y, __fmaf_rn(v.z, v.z, __fmaf_rn(v.w, v.w, acc))));
}

template <bool F32>
__global__ void __launch_bounds__(256) block_embed_kernel(const uint16_t *__restrict__ table, const uint32_t *__restrict__ tokens, uint32_t n, float *__restrict__ x,
                                                         size_t x_stride, const Act out) {
    const uint32_t t = blockIdx.y, k = blockIdx.x * 256 + threadIdx.x;
    pdl_wait();
    pdl_trigger();
    if (k >= n) return;
    const float v = bf16_bits_to_f32(__ldg(table + (size_t)__ldcg(tokens + t) * n + k));
    x[t * x_stride + k] = v;
    act_store<F32>(out, t, k, v);
}

template <bool F32, bool ADD, bool PRE>
__global__ void __launch_bounds__(1024) block_norm_kernel(const NormArgs a) {
    __shared__ float scratch[32];
    const uint32_t t = blockIdx.x, n = a.n;
    float *xr = a.x + t * a.x_stride, *yr = ADD ? a.y + t * a.y_stride : nullptr;
    pdl_wait();
    pdl_trigger();
    const uint32_t step = blockDim.x * 4, k_first = threadIdx.x * 4;
    float4 v0 = make_float4(0, 0, 0, 0), x0 = v0;          // the first step's values stay in registers
    float ss[1] = {0.0f};
    if (ADD) {
        auto sublayer = [&](uint32_t k) {
            float4 v = load4(yr, k, n);
            if (a.top > 0) {
                for (uint32_t i = 0; i < a.top; ++i) {
                    const float w = __ldcg(a.weight + t * a.top + i);
                    const float4 q = load4(a.pairs + (size_t)__ldcg(a.row + t * a.top + i) * a.pair_stride, k, n);
                    v = make_float4(__fmaf_rn(w, q.x, v.x), __fmaf_rn(w, q.y, v.y), __fmaf_rn(w, q.z, v.z), __fmaf_rn(w, q.w, v.w));
                }
                *reinterpret_cast<float4 *>(yr + k) = v;
            }
            return v;
        };
        if (k_first < n) { x0 = load4(xr, k_first, n); v0 = sublayer(k_first); ss[0] = sq4(v0, ss[0]); }
        for (uint32_t k = k_first + step; k < n; k += step) ss[0] = sq4(sublayer(k), ss[0]);
        block_sum<1>(ss, scratch);
        const float inv = 1.0f / sqrtf(ss[0] / (float)n + a.eps);
        ss[0] = 0.0f;
        for (uint32_t k = k_first; k < n; k += step) {
            const float4 v = k == k_first ? v0 : load4(yr, k, n), o = k == k_first ? x0 : load4(xr, k, n), g = __ldg(reinterpret_cast<const float4 *>(a.post + k));
            const float4 r = make_float4(o.x + a.mult * (v.x * inv * g.x), o.y + a.mult * (v.y * inv * g.y), o.z + a.mult * (v.z * inv * g.z), o.w + a.mult * (v.w * inv * g.w));
            *reinterpret_cast<float4 *>(xr + k) = r;
            if (!PRE) act_store4<F32>(a.out, t, k, n, r);
            if (PRE) ss[0] = sq4(r, ss[0]);
            if (k == k_first) x0 = r;
        }
    } else {
        if (k_first < n) { x0 = load4(xr, k_first, n); ss[0] = sq4(x0, ss[0]); }
        for (uint32_t k = k_first + step; k < n; k += step) ss[0] = sq4(load4(xr, k, n), ss[0]);
    }
    if (PRE) {
        block_sum<1>(ss, scratch);
        const float inv = 1.0f / sqrtf(ss[0] / (float)n + a.eps);
        for (uint32_t k = k_first; k < n; k += step) {
            const float4 v = k == k_first ? x0 : load4(xr, k, n), g = __ldg(reinterpret_cast<const float4 *>(a.pre + k));
            act_store4<F32>(a.out, t, k, n, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
        }
    }
}

// A cluster of `cs` CTAs per token; CTA r holds the panels [r np / cs, (r + 1) np / cs) of the vector.  Two exchanges over
// distributed shared memory: the sublayer's sum of squares together with the partial gate products - of x and of y w apart, so
// that the products need not wait for the norm: gate (x + y w / rms) = gate x + gate (y w) / rms - and the token input's sum of
// squares.
// The CTA's share of both weight matrices is bulk-copied to shared memory before the dependency wait (STAGED: bf16 panels that
// fit), so after the wait only the two vectors come from global memory.
constexpr uint32_t NS_THREADS = 256;
constexpr uint32_t NS_MAX_CS = 8;
constexpr uint32_t NS_WAIT_LIMIT = 1u << 22;

__host__ __device__ inline uint32_t ns_slice_panels(uint32_t np, uint32_t cs) { return (np + cs - 1) / cs; }
inline size_t ns_vec_smem(uint32_t n, uint32_t dim, uint32_t cs) {
    const uint32_t slice = ns_slice_panels((n + 63) / 64, cs) * 64, dp = (dim + 63) / 64 * 64;
    return (((size_t)2 * slice + dp + (size_t)2 * cs * dim) * 4 + 127) & ~(size_t)127;
}
inline size_t ns_weight_smem(uint32_t n, uint32_t dim, uint32_t cs) {
    const uint32_t sp = ns_slice_panels((n + 63) / 64, cs), dp = (dim + 63) / 64;
    return (size_t)sp * dim * 128 + (size_t)dp * sp * 64 * 128;
}

template <bool F32, bool STAGED>
__global__ void __launch_bounds__(NS_THREADS) norm_side_kernel(float *__restrict__ x, size_t x_stride, const float *__restrict__ y, size_t y_stride, const float *__restrict__ w,
                                                              uint32_t n, float eps, const SideArgs sd, const Act out, uint32_t weights_at, uint32_t *__restrict__ err_flag) {
    extern __shared__ __align__(128) float sm[];
    __shared__ float scratch[32], slot_a[NS_MAX_CS], slot_b[NS_MAX_CS];
    __shared__ __align__(8) uint64_t bar_w;
    const uint32_t cs = cluster_size(), me = cluster_rank(), t = blockIdx.x / cs, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t np = (n + 63) / 64, sp = ns_slice_panels(np, cs), p0 = min(np, me * sp), p1 = min(np, p0 + sp);
    const uint32_t slice = sp * 64, dim = sd.dim, dp = (dim + 63) / 64 * 64;
    float *s_x = sm, *s_y = s_x + slice, *s_g = s_y + slice, *s_part = s_g + dp;      // s_part [cs][2 dim]: written by the peers
    const uint32_t k0 = p0 * 64, k1 = min(n, p1 * 64);
    DenseView gate = sd.gate, proj = sd.proj;
    const uint32_t bar = (uint32_t)__cvta_generic_to_shared(&bar_w);
    if (STAGED) {
        uint8_t *s_w = reinterpret_cast<uint8_t *>(sm) + weights_at;
        const uint32_t mine = p1 - p0, sw = (uint32_t)__cvta_generic_to_shared(s_w);
        if (tid == 0) {
            mbar_init(bar, 1);
            fence_mbar_init();
            mbar_expect_tx(bar, mine * dim * 128 + proj.panels * mine * 64 * 128);
            const uint8_t *gb = static_cast<const uint8_t *>(sd.gate.base), *pb = static_cast<const uint8_t *>(sd.proj.base);
            for (uint32_t p = 0; p < mine; ++p) bulk_g2s(sw + p * dim * 128, gb + (size_t)(p0 + p) * sd.gate.rows_pad * 128, dim * 128, bar);
            for (uint32_t q = 0; q < proj.panels && mine > 0; ++q)
                bulk_g2s(sw + mine * dim * 128 + q * mine * 64 * 128, pb + ((size_t)q * sd.proj.rows_pad + k0) * 128, mine * 64 * 128, bar);
        }
        gate.base = s_w; gate.rows_pad = dim;
        proj.base = s_w + mine * dim * 128; proj.rows_pad = mine * 64;
    }
    for (uint32_t i = tid; i < 2 * slice; i += NS_THREADS) s_x[i] = 0.0f;      // s_x and s_y
    for (uint32_t i = tid; i < dp; i += NS_THREADS) s_g[i] = 0.0f;
    float w_first = 0.0f, n_first = 0.0f;       // the norm weights of the thread's first element
    if (k0 + tid < k1) { w_first = __ldg(w + k0 + tid); n_first = __ldg(sd.norm + k0 + tid); }
    if (cs > 1) cluster_sync_all();             // every CTA of the cluster runs before its shared memory is written from outside
    pdl_wait();
    pdl_trigger();
    float *xr = x + t * x_stride;
    const float *yr = y + t * y_stride;
    const uint16_t *e = sd.table + (size_t)__ldcg(sd.tokens + t) * sd.table_stride + sd.offset;
    const float e_first = tid < dim ? bf16_bits_to_f32(__ldg(e + tid)) : 0.0f;
    float ss[1] = {0.0f};
    for (uint32_t k = k0 + tid; k < k1; k += NS_THREADS) {
        const float v = __ldcg(yr + k);
        s_x[k - k0] = __ldcg(xr + k);
        s_y[k - k0] = v * (k == k0 + tid ? w_first : __ldg(w + k));
        ss[0] = __fmaf_rn(v, v, ss[0]);
    }
    if (STAGED) {
        bool ok = false;
        for (uint32_t spin = 0; spin < NS_WAIT_LIMIT && !ok; ++spin) ok = mbar_try_wait(bar, 0u);
        if (!ok && err_flag != nullptr) atomicExch(err_flag, 1u);
    }
    block_sum<1>(ss, scratch);                  // its barriers also publish s_x and s_y
    // partial gate products of the slice: eight lanes per row, four rows per warp and step
    const uint32_t sub = lane & 7u, q0 = STAGED ? 0u : p0, q1 = STAGED ? p1 - p0 : p1;
    // (loops kept rolled: the kernel runs its code once per launch, and instruction fetch is what unrolled copies cost)
#pragma unroll 1
    for (uint32_t r0 = warp * 4; r0 < dim; r0 += NS_THREADS / 8) {
        const uint32_t r = r0 + (lane >> 3), rr = min(r, dim - 1);
        float dx = 0.0f, dy = 0.0f;
        if (STAGED) {
            const uint4 *q = static_cast<const uint4 *>(gate.base) + (size_t)rr * 8 + (sub ^ (rr & 7u));
#pragma unroll 1
            for (uint32_t k = sub * 8; k < (p1 - p0) * PANEL; k += PANEL, q += (size_t)dim * 8) {
                const uint4 v = *q;
                dx = dot8(v, s_x + k, dx);
                dy = dot8(v, s_y + k, dy);
            }
#pragma unroll
            for (int m = 1; m < 8; m <<= 1) { dx = __fadd_rn(dx, __shfl_xor_sync(0xffffffffu, dx, m)); dy = __fadd_rn(dy, __shfl_xor_sync(0xffffffffu, dy, m)); }
        } else {
            dx = row_dot8<F32>(gate, rr, q0, q1, s_x, sub);
            dy = row_dot8<F32>(gate, rr, q0, q1, s_y, sub);
        }
        if (r < dim && sub < cs) { st_cluster_f32(s_part + ((size_t)me * 2) * dim + r, sub, dx); st_cluster_f32(s_part + ((size_t)me * 2 + 1) * dim + r, sub, dy); }
    }
    if (cs == 1) __syncthreads();
    cluster_sum<1>(ss, slot_a);                 // its barrier also publishes the partial products
    const float inv = rsqrtf(ss[0] / (float)n + eps);
    for (uint32_t i = tid; i < dim; i += NS_THREADS) {
        float zx = 0.0f, zy = 0.0f;
        for (uint32_t r = 0; r < cs; ++r) { zx = __fadd_rn(zx, s_part[((size_t)r * 2) * dim + i]); zy = __fadd_rn(zy, s_part[((size_t)r * 2 + 1) * dim + i]); }
        s_g[i] = gelu_tanh(__fmaf_rn(zy, inv, zx)) * (i == tid ? e_first : bf16_bits_to_f32(__ldg(e + i)));
    }
    for (uint32_t k = tid; k < k1 - k0 && k1 > k0; k += NS_THREADS) s_x[k] = __fmaf_rn(s_y[k], inv, s_x[k]);
    __syncthreads();
    float s2[1] = {0.0f};
    const uint32_t row_off = STAGED ? k0 : 0u;
#pragma unroll 1
    for (uint32_t r0 = k0 + warp * 4; r0 < k1; r0 += NS_THREADS / 8) {
        const uint32_t r = r0 + (lane >> 3);
        const float d = row_dot8<F32, STAGED>(proj, min(r, k1 - 1) - row_off, 0, proj.panels, s_g, sub);
        if (r < k1 && sub == 0) { s_y[r - k0] = d; s2[0] = __fmaf_rn(d, d, s2[0]); }
    }
    block_sum<1>(s2, scratch);
    cluster_sum<1>(s2, slot_b);
    const float inv2 = rsqrtf(s2[0] / (float)n + eps);
    for (uint32_t k = k0 + tid; k < k1; k += NS_THREADS) {
        const float v = s_x[k - k0] + s_y[k - k0] * inv2 * (k == k0 + tid ? n_first : __ldg(sd.norm + k));
        xr[k] = v;
        act_store<F32>(out, t, k, v);
    }
    if (cs > 1) cluster_sync_all();             // no CTA leaves while a peer may still write to it
}

template <bool F32>
__global__ void __launch_bounds__(256) side_gelu_kernel(const float *__restrict__ z, size_t z_stride, const SideArgs sd, uint32_t n_tok, const Act out) {
    const uint32_t i = blockIdx.x * 256 + threadIdx.x;
    pdl_wait();
    pdl_trigger();
    if (i >= n_tok * sd.dim) return;
    const uint32_t t = i / sd.dim, k = i % sd.dim;
    const float e = bf16_bits_to_f32(__ldg(sd.table + (size_t)__ldcg(sd.tokens + t) * sd.table_stride + sd.offset + k));
    act_store<F32>(out, t, k, gelu_tanh(__ldcg(z + t * z_stride + k)) * e);
}

template <bool F32>
__global__ void __launch_bounds__(256) polynorm_kernel(const float *__restrict__ z, size_t z_stride, uint32_t n, const float *__restrict__ coef, float eps, const Act out) {
    __shared__ float scratch[96], slots[3 * NS_MAX_CS];
    const uint32_t cs = cluster_size(), me = cluster_rank(), t = blockIdx.x / cs;
    const uint32_t np = (n + 63) / 64, p0 = min(np, me * ns_slice_panels(np, cs)), p1 = min(np, p0 + ns_slice_panels(np, cs));
    const uint32_t k0 = p0 * 64 + threadIdx.x * 4, k1 = min(n, p1 * 64);
    const float ca = __ldg(coef), cb = __ldg(coef + 1), cc = __ldg(coef + 2), ce = __ldg(coef + 3);
    if (cs > 1) cluster_sync_all();
    pdl_wait();
    pdl_trigger();
    const float *zr = z + t * z_stride;
    float m[3] = {0.0f, 0.0f, 0.0f};             // sums of z^2, z^4, z^6
    constexpr uint32_t KEEP = 8;
    float4 keep[KEEP];                            // the first values of the thread stay in registers
#pragma unroll
    for (uint32_t i = 0; i < KEEP; ++i) {
        const uint32_t k = k0 + i * 1024;
        if (k < k1) keep[i] = load4(zr, k, n);
    }
    auto power = [&](const float4 &v) {
        const float e[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float q = e[i] * e[i], q2 = q * q; m[0] += q; m[1] += q2; m[2] = __fmaf_rn(q2, q, m[2]); }
    };
#pragma unroll
    for (uint32_t i = 0; i < KEEP; ++i)
        if (k0 + i * 1024 < k1) power(keep[i]);
    for (uint32_t k = k0 + KEEP * 1024; k < k1; k += 1024) power(load4(zr, k, n));
    block_sum<3>(m, scratch);
    cluster_sum<3>(m, slots);
    const float fn = (float)n, f1 = ca / sqrtf(m[0] / fn + eps), f2 = cb / sqrtf(m[1] / fn + eps), f3 = cc / sqrtf(m[2] / fn + eps);
    auto value = [&](float v) { return __fmaf_rn(v, __fmaf_rn(v, __fmaf_rn(v, f3, f2), f1), ce); };
    auto store = [&](uint32_t k, const float4 &v) { act_store4<F32>(out, t, k, n, make_float4(value(v.x), value(v.y), value(v.z), value(v.w))); };
#pragma unroll
    for (uint32_t i = 0; i < KEEP; ++i)
        if (k0 + i * 1024 < k1) store(k0 + i * 1024, keep[i]);
    for (uint32_t k = k0 + KEEP * 1024; k < k1; k += 1024) store(k, load4(zr, k, n));
    if (cs > 1) cluster_sync_all();
}

uint32_t cluster_for(uint32_t np, uint32_t n_tok) {       // CTAs per token: few tokens spread over the SMs
    uint32_t cs = 1;
    while (cs < NS_MAX_CS && cs * 2 <= np && cs * 2 * n_tok <= 160) cs *= 2;
    return cs;
}

}  // namespace

cudaError_t launch_block_embed(cudaStream_t s, bool f32, const uint16_t *table, const uint32_t *tokens, uint32_t n, float *x, size_t x_stride, const Act &out,
                               uint32_t n_tok, bool pdl) {
    return launch_kernel(f32 ? block_embed_kernel<true> : block_embed_kernel<false>, dim3((n + 255) / 256, n_tok), dim3(256), 0, s, pdl, table, tokens, n, x, x_stride, out);
}

cudaError_t launch_block_norm(cudaStream_t s, bool f32, const NormArgs &a, uint32_t n_tok, bool pdl) {
    if (a.y == nullptr && a.pre == nullptr) return cudaErrorInvalidValue;
    const uint32_t threads = std::min(n_tok > 64 ? 512u : 1024u, std::max(32u, ((a.n + 3) / 4 + 31u) & ~31u));
    auto k = f32 ? (a.y == nullptr ? block_norm_kernel<true, false, true> : a.pre == nullptr ? block_norm_kernel<true, true, false> : block_norm_kernel<true, true, true>)
                 : (a.y == nullptr ? block_norm_kernel<false, false, true> : a.pre == nullptr ? block_norm_kernel<false, true, false> : block_norm_kernel<false, true, true>);
    return launch_kernel(k, dim3(n_tok), dim3(threads), 0, s, pdl, a);
}

bool norm_side_fits(uint32_t n, uint32_t dim) { return ns_vec_smem(n, dim, 1) <= 200 * 1024; }

cudaError_t launch_norm_side(cudaStream_t s, bool f32, float *x, size_t x_stride, const float *y, size_t y_stride, const float *w, uint32_t n, float eps,
                             const SideArgs &side, const Act &out, uint32_t n_tok, uint32_t *err_flag, bool pdl) {
    const uint32_t cs = cluster_for((n + 63) / 64, n_tok);
    const size_t vec = ns_vec_smem(n, side.dim, cs), all = vec + ns_weight_smem(n, side.dim, cs);
    const bool staged = !f32 && all <= 200 * 1024;
    auto k = f32 ? norm_side_kernel<true, false> : staged ? norm_side_kernel<false, true> : norm_side_kernel<false, false>;
    const size_t smem = staged ? all : vec;
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(k), smem);
    if (e != cudaSuccess) return e;
    return launch_cluster(k, dim3(cs * n_tok), dim3(NS_THREADS), smem, s, pdl, cs, x, x_stride, y, y_stride, w, n, eps, side, out, (uint32_t)vec, err_flag);
}

cudaError_t launch_side_gelu(cudaStream_t s, bool f32, const float *z, size_t z_stride, const SideArgs &side, const Act &out, uint32_t n_tok, bool pdl) {
    return launch_kernel(f32 ? side_gelu_kernel<true> : side_gelu_kernel<false>, dim3((n_tok * side.dim + 255) / 256), dim3(256), 0, s, pdl, z, z_stride, side, n_tok, out);
}

cudaError_t launch_polynorm(cudaStream_t s, bool f32, const float *z, size_t z_stride, uint32_t n, const float *coef, float eps, const Act &out, uint32_t n_tok, bool pdl) {
    const uint32_t cs = cluster_for((n + 63) / 64, n_tok);
    return launch_cluster(f32 ? polynorm_kernel<true> : polynorm_kernel<false>, dim3(cs * n_tok), dim3(256), 0, s, pdl, cs, z, z_stride, n, coef, eps, out);
}

}  // namespace k2t
