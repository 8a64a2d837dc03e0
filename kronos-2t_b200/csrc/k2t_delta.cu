// Generalized delta rule of the block engine (k2t_block_kernels.h), fp32 throughout: per head a state S [key][value] with
//   S_t = diag(w) S_(t-1) - (a u)(u^T S_(t-1)) + k v^T,   o_t = S_t^T r,
// w the decay and a the removal rate per key channel, u the unit key.  Columns of S do not meet, so a column group of a head is
// an independent chain.
//   * delta_step_kernel (one token): a cluster per head.  The state is requested before the dependency wait (only the same
//     layer's previous step wrote it), then coefficients, recurrence, per-head norm, output gate and the activation of the output
//     projection in one launch.
//   * prompts: delta_prep_kernel writes the coefficients of every head and group of four tokens as one record,
//     delta_scan_kernel walks the groups - a warp holds two or four columns, its lanes share the keys - with the records streamed through
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
// A cluster of drow / 32 CTAs per head, CTA = 32 columns: thread = (four columns, KPS = drow / 32 keys).  Every CTA makes the
// head's coefficients; only the sum of squares of o crosses the cluster.
constexpr uint32_t ST_THREADS = 256, ST_COLS = 32, ST_SLICES = ST_THREADS / (ST_COLS / 4);
constexpr uint32_t ST_WAIT_LIMIT = 1u << 22;
inline size_t step_vec_smem(uint32_t drow, uint32_t rank_pad) { return (((size_t)5 * drow + ST_COLS + ST_SLICES * ST_COLS + rank_pad) * 4 + 127) & ~(size_t)127; }

template <bool F32, int KPS, bool STAGED>
__global__ void __launch_bounds__(ST_THREADS) delta_step_kernel(const DeltaArgs a, uint32_t weights_at) {
    extern __shared__ __align__(128) float sm[];
    __shared__ float scratch[32], slots[8];
    __shared__ __align__(8) uint64_t bar_w;
    constexpr uint32_t D = 32 * KPS, SLICES = ST_SLICES;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, cs = cluster_size(), me = cluster_rank(), h = blockIdx.x / cs, dim = a.dim;
    const uint32_t q = tid & 7u, sl = tid >> 3, col0 = me * ST_COLS, rank_pad = (a.rank + 63) / 64 * 64;
    float *s_w = sm, *s_au = s_w + D, *s_u = s_au + D, *s_k = s_u + D, *s_r = s_k + D, *s_v = s_r + D, *s_red = s_v + ST_COLS, *s_t = s_red + SLICES * ST_COLS;
    float4 st[KPS];
    float *state = a.state + (size_t)h * D * D + (size_t)(sl * KPS) * D + col0 + q * 4;
#pragma unroll
    for (uint32_t i = 0; i < KPS; ++i) st[i] = __ldcg(reinterpret_cast<const float4 *>(state + (size_t)i * D));
    for (uint32_t i = tid; i < 5 * D + ST_COLS; i += ST_THREADS) sm[i] = 0.0f;
    for (uint32_t i = tid; i < rank_pad; i += ST_THREADS) s_t[i] = 0.0f;
    DenseView decay = a.decay;
    const uint32_t bar = (uint32_t)__cvta_generic_to_shared(&bar_w), row0 = h * dim & ~7u;          // the head's rows, from a whole swizzle octet on
    if (STAGED) {       // the head's rows of the decay product: weights, copied while the predecessor runs
        uint8_t *s_d = reinterpret_cast<uint8_t *>(sm) + weights_at;
        const uint32_t rows = h * dim + dim - row0;
        if (tid == 0) {
            mbar_init(bar, 1);
            fence_mbar_init();
            mbar_expect_tx(bar, rows * 128 * decay.panels);
            for (uint32_t p = 0; p < decay.panels; ++p)
                bulk_g2s((uint32_t)__cvta_generic_to_shared(s_d) + p * rows * 128, static_cast<const uint8_t *>(a.decay.base) + ((size_t)p * a.decay.rows_pad + row0) * 128, rows * 128, bar);
        }
        decay.base = s_d; decay.rows_pad = rows;
    }
    const float norm_w = tid < ST_COLS && col0 + tid < dim ? __ldg(a.norm + h * dim + col0 + tid) : 0.0f;
    if (cs > 1) cluster_sync_all();             // every CTA of the cluster runs before its shared memory is written from outside
    pdl_wait();
    pdl_trigger();
    __syncthreads();
    const uint32_t HD = a.heads * dim;
    const float *in = a.in + h * dim;
    float kk[1] = {0.0f}, rate = 0.0f, gate = 0.0f, bias = 0.0f;
    if (tid < dim) {                            // dim <= 256 = threads
        const float k = __ldcg(in + HD + tid);
        s_r[tid] = __ldcg(in + tid);
        s_k[tid] = k;
        rate = __ldcg(in + 4 * HD + tid) + __ldg(a.rate_bias + h * dim + tid);
        bias = __ldg(a.decay_bias + h * dim + tid);
        kk[0] = k * k;
    }
    if (tid < ST_COLS && col0 + tid < dim) { s_v[tid] = __ldcg(in + 2 * HD + col0 + tid); gate = __ldcg(in + 3 * HD + col0 + tid); }
    for (uint32_t i = tid; i < a.rank; i += ST_THREADS) s_t[i] = tanhf(__ldcg(a.in + 5 * HD + i));
    block_sum<1>(kk, scratch);                          // its barriers also publish s_t, s_k
    const float inv_k = 1.0f / sqrtf(kk[0] + a.unit_eps);
    if (tid < dim) { const float u = s_k[tid] * inv_k; s_u[tid] = u; s_au[tid] = sigmoidf(rate) * u; }
    if (STAGED) {
        bool ok = false;
        for (uint32_t spin = 0; spin < ST_WAIT_LIMIT && !ok; ++spin) ok = mbar_try_wait(bar, 0u);
        if (!ok && a.err_flag != nullptr) atomicExch(a.err_flag, 1u);
    }
    const uint32_t sub = lane & 7u;
#pragma unroll 1
    for (uint32_t r0 = warp * 4; r0 < dim; r0 += ST_THREADS / 8) {
        const uint32_t i = r0 + (lane >> 3), c = h * dim + min(i, dim - 1);
        const float z = row_dot8<F32, STAGED>(decay, STAGED ? c - row0 : c, 0, decay.panels, s_t, sub);
        if (i < dim && sub == 0) s_w[i] = z;
    }
    __syncthreads();
    if (tid < dim) s_w[tid] = decay_minus_one(a.decay_scale, s_w[tid] + bias);
    __syncthreads();
    float4 c = make_float4(0, 0, 0, 0);
#pragma unroll
    for (uint32_t i = 0; i < KPS; ++i) {
        const float u = s_u[sl * KPS + i];
        c.x = __fmaf_rn(u, st[i].x, c.x); c.y = __fmaf_rn(u, st[i].y, c.y); c.z = __fmaf_rn(u, st[i].z, c.z); c.w = __fmaf_rn(u, st[i].w, c.w);
    }
    *reinterpret_cast<float4 *>(s_red + sl * ST_COLS + q * 4) = c;
    __syncthreads();
    c = make_float4(0, 0, 0, 0);
#pragma unroll 8
    for (uint32_t s = 0; s < SLICES; ++s) {
        const float4 p = *reinterpret_cast<const float4 *>(s_red + s * ST_COLS + q * 4);
        c.x += p.x; c.y += p.y; c.z += p.z; c.w += p.w;
    }
    const float4 v = *reinterpret_cast<const float4 *>(s_v + q * 4);
    float4 o = make_float4(0, 0, 0, 0);
#pragma unroll
    for (uint32_t i = 0; i < KPS; ++i) {
        const uint32_t key = sl * KPS + i;
        const float w = s_w[key], au = -s_au[key], k = s_k[key], r = s_r[key];
        st[i].x = __fmaf_rn(au, c.x, __fmaf_rn(w, st[i].x, __fmaf_rn(k, v.x, st[i].x))); st[i].y = __fmaf_rn(au, c.y, __fmaf_rn(w, st[i].y, __fmaf_rn(k, v.y, st[i].y)));
        st[i].z = __fmaf_rn(au, c.z, __fmaf_rn(w, st[i].z, __fmaf_rn(k, v.z, st[i].z))); st[i].w = __fmaf_rn(au, c.w, __fmaf_rn(w, st[i].w, __fmaf_rn(k, v.w, st[i].w)));
        o.x = __fmaf_rn(r, st[i].x, o.x); o.y = __fmaf_rn(r, st[i].y, o.y); o.z = __fmaf_rn(r, st[i].z, o.z); o.w = __fmaf_rn(r, st[i].w, o.w);
        *reinterpret_cast<float4 *>(state + (size_t)i * D) = st[i];
    }
    __syncthreads();                                    // every thread has read the partial sums
    *reinterpret_cast<float4 *>(s_red + sl * ST_COLS + q * 4) = o;
    __syncthreads();
    float so[1] = {0.0f}, mine = 0.0f;
    if (tid < ST_COLS) {
#pragma unroll 8
        for (uint32_t s = 0; s < SLICES; ++s) mine += s_red[s * ST_COLS + tid];          // columns beyond dim hold zeros
        so[0] = warp_sum(mine * mine);
        if (tid == 0) scratch[0] = so[0];
    }
    __syncthreads();
    so[0] = scratch[0];
    cluster_sum<1>(so, slots);
    const float inv = 1.0f / sqrtf(so[0] / (float)dim + a.eps);
    if (tid < ST_COLS && col0 + tid < dim) act_store<F32>(a.out, 0, h * dim + col0 + tid, mine * inv * norm_w * sigmoidf(gate));
    if (cs > 1) cluster_sync_all();                     // no CTA leaves while a peer may still write to it
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

constexpr uint32_t SC_STAGES = 3;
constexpr uint32_t SC_WAIT_LIMIT = 1u << 22;
__host__ __device__ constexpr uint32_t stage_groups(uint32_t drow) { return drow >= 256 ? 1u : 256u / drow; }

// Twice N values per lane (N = 8 or 16) summed over the warp side by side: lane l returns the sums of a[l N / 32] and b[l N / 32]
// (an exchange halves the values per step).
template <int N> __device__ __forceinline__ float2 warp_sum_many(float (&a)[N], float (&b)[N], uint32_t lane) {
    constexpr int SPREAD = 32 / N;
#pragma unroll
    for (int w = N / 2; w > 0; w >>= 1) {
        const bool up = (lane & (w * SPREAD)) != 0;
#pragma unroll
        for (int i = 0; i < w; ++i) {
            const float ga = up ? a[i] : a[i + w], ka = up ? a[i + w] : a[i], gb = up ? b[i] : b[i + w], kb = up ? b[i + w] : b[i];
            a[i] = __fadd_rn(ka, __shfl_xor_sync(0xffffffffu, ga, w * SPREAD));
            b[i] = __fadd_rn(kb, __shfl_xor_sync(0xffffffffu, gb, w * SPREAD));
        }
    }
    float ra = a[0], rb = b[0];
#pragma unroll
    for (int m = SPREAD / 2; m > 0; m >>= 1) { ra = __fadd_rn(ra, __shfl_xor_sync(0xffffffffu, ra, m)); rb = __fadd_rn(rb, __shfl_xor_sync(0xffffffffu, rb, m)); }
    return make_float2(ra, rb);
}
__device__ __forceinline__ uint64_t lds64(uint32_t saddr) {        // kept in program order: a group's loads are issued ahead of its reductions
    uint64_t v;
    asm volatile("ld.shared.b64 %0, [%1];" : "=l"(v) : "r"(saddr) : "memory");
    return v;
}

// CTA = four warps, warp = NC (two or four) columns of a head; the 32 lanes share the keys: lane l holds the key pairs
// 2 (32 i + l), i < KP (drow = 64 KP), so a record vector is read once per warp, 256 consecutive bytes per load.  Two columns
// give the SMs twice the warps to hide latencies with where there are few heads, four halve the shared-memory reads.
template <int KP, int NC>
__global__ void __launch_bounds__(128) delta_scan_kernel(const float *__restrict__ rec, uint32_t n_tok, float *__restrict__ state, float *__restrict__ o, uint32_t heads,
                                                        uint32_t *__restrict__ err_flag) {
    extern __shared__ __align__(128) float ring[];
    __shared__ __align__(8) uint64_t bars[SC_STAGES];
    constexpr uint32_t D = 64 * KP, GF = group_floats(D), SG = stage_groups(D), STAGE = SG * GF;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, col = (blockIdx.x * 4 + warp) * NC;
    const uint32_t bar = (uint32_t)__cvta_generic_to_shared(bars), rb = (uint32_t)__cvta_generic_to_shared(ring);
    const uint32_t groups = (n_tok + GROUP - 1) / GROUP, chunks = (groups + SG - 1) / SG;
    const float *src = rec + (size_t)h * groups * GF;
    if (tid == 0) {
        for (uint32_t i = 0; i < SC_STAGES; ++i) mbar_init(bar + 8 * i, 1);
        fence_mbar_init();
    }
    float *sp = state + (size_t)h * D * D + col;
    uint64_t s[NC][KP];
#pragma unroll
    for (int i = 0; i < KP; ++i) {
        const float *q = sp + (size_t)((i * 32 + lane) * 2) * D;
#pragma unroll
        for (int c = 0; c < NC; c += 2) {
            const float2 e = __ldcg(reinterpret_cast<const float2 *>(q + c)), f = __ldcg(reinterpret_cast<const float2 *>(q + D + c));
            s[c][i] = pk(e.x, f.x); s[c + 1][i] = pk(e.y, f.y);
        }
    }
    pdl_wait();
    pdl_trigger();
    __syncthreads();
    float oo[GROUP * NC];                       // outputs of the group before, not reduced yet
#pragma unroll
    for (int i = 0; i < (int)GROUP * NC; ++i) oo[i] = 0.0f;
    uint32_t tok_o = n_tok;                     // its first token; n_tok = none
    auto store = [&](uint32_t tok0, float sum) {
        constexpr uint32_t LPV = 32 / (GROUP * NC);          // lanes that hold the same value
        const uint32_t tok = tok0 + (lane >> 3);
        if (lane % LPV == 0 && tok < n_tok) o[((size_t)tok * heads + h) * D + col + (lane / LPV) % NC] = sum;
    };
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
        uint32_t sa = rb + (c % SC_STAGES) * STAGE * 4 + lane * 8;
#pragma unroll 1
        for (uint32_t gi = 0; gi < n; ++gi, at += GF, sa += GF * 4) {
            uint64_t part[5][GROUP][KP];        // U, then w - 1, a u, k, r
#pragma unroll
            for (int j = 0; j < 5; ++j)
#pragma unroll
                for (uint32_t t = 0; t < GROUP; ++t)
#pragma unroll
                    for (int i = 0; i < KP; ++i) part[j][t][i] = lds64(sa + ((t * 6 + (j == 0 ? 2 : j <= 2 ? j - 1 : j)) * (D / 2) + i * 32) * 8);
            float d[GROUP * NC], v[GROUP * NC];
#pragma unroll
            for (uint32_t t = 0; t < GROUP; ++t) {
                uint64_t p[NC];
#pragma unroll
                for (int i = 0; i < KP; ++i)
#pragma unroll
                    for (int c2 = 0; c2 < NC; ++c2) p[c2] = fma2(part[0][t][i], s[c2][i], i == 0 ? 0ull : p[c2]);
#pragma unroll
                for (int c2 = 0; c2 < NC; c2 += 2) {
                    const float2 e = *reinterpret_cast<const float2 *>(at + (t * 6 + 5) * D + col + c2);
                    v[t * NC + c2] = e.x; v[t * NC + c2 + 1] = e.y;
                }
#pragma unroll
                for (int c2 = 0; c2 < NC; ++c2) { float e0, e1; upk(p[c2], e0, e1); d[t * NC + c2] = __fadd_rn(e0, e1); }
            }
            // the products of this group and the outputs of the one before are reduced side by side
            const float2 sums = warp_sum_many<GROUP * NC>(d, oo, lane);
            store(tok_o, sums.y);
            tok_o = (c * SG + gi) * GROUP;
#pragma unroll
            for (int i = 0; i < (int)GROUP * NC; ++i) d[i] = __shfl_sync(0xffffffffu, sums.x, 32 / (GROUP * NC) * i);
            const float *gh = at + GROUP * 6 * D;
#pragma unroll
            for (uint32_t t = 1; t < GROUP; ++t)
#pragma unroll
                for (uint32_t q = 0; q < t; ++q) {
                    const float g = gh[t * (t - 1) / 2 + q], hh = -gh[6 + t * (t - 1) / 2 + q];
#pragma unroll
                    for (int c2 = 0; c2 < NC; ++c2) d[t * NC + c2] = __fmaf_rn(hh, d[q * NC + c2], __fmaf_rn(g, v[q * NC + c2], d[t * NC + c2]));
                }
#pragma unroll
            for (uint32_t t = 0; t < GROUP; ++t) {
                uint64_t v2[NC], c2n[NC], p[NC];
#pragma unroll
                for (int c2 = 0; c2 < NC; ++c2) { v2[c2] = pk(v[t * NC + c2], v[t * NC + c2]); c2n[c2] = pk(-d[t * NC + c2], -d[t * NC + c2]); }
#pragma unroll
                for (int i = 0; i < KP; ++i)
#pragma unroll
                    for (int c2 = 0; c2 < NC; ++c2) {
                        s[c2][i] = fma2(part[2][t][i], c2n[c2], fma2(part[1][t][i], s[c2][i], fma2(part[3][t][i], v2[c2], s[c2][i])));
                        p[c2] = fma2(part[4][t][i], s[c2][i], i == 0 ? 0ull : p[c2]);
                    }
#pragma unroll
                for (int c2 = 0; c2 < NC; ++c2) { float e0, e1; upk(p[c2], e0, e1); oo[t * NC + c2] = __fadd_rn(e0, e1); }
            }
        }
        __syncthreads();                        // the stage is free
        if (tid == 0 && c + SC_STAGES < chunks) request(c + SC_STAGES);
    }
    {
        float none[GROUP * NC];
#pragma unroll
        for (int i = 0; i < (int)GROUP * NC; ++i) none[i] = 0.0f;
        store(tok_o, warp_sum_many<GROUP * NC>(none, oo, lane).y);
    }
#pragma unroll
    for (int i = 0; i < KP; ++i) {
        float *q = sp + (size_t)((i * 32 + lane) * 2) * D;
#pragma unroll
        for (int c = 0; c < NC; c += 2) {
            float2 e, f;
            upk(s[c][i], e.x, f.x); upk(s[c + 1][i], e.y, f.y);
            *reinterpret_cast<float2 *>(q + c) = e;
            *reinterpret_cast<float2 *>(q + D + c) = f;
        }
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

template <int KP, int NC> cudaError_t scan_nc(cudaStream_t s, const DeltaArgs &a, uint32_t n_tok, bool pdl) {
    constexpr size_t smem = (size_t)SC_STAGES * stage_groups(64 * KP) * group_floats(64 * KP) * 4;
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(delta_scan_kernel<KP, NC>), smem);
    if (e != cudaSuccess) return e;
    return launch_kernel(delta_scan_kernel<KP, NC>, dim3(64 * KP / (4 * NC), a.heads), dim3(128), smem, s, pdl, a.rec, n_tok, a.state, a.o, a.heads, a.err_flag);
}
template <int KP> cudaError_t scan_kp(cudaStream_t s, const DeltaArgs &a, uint32_t n_tok, int sm_count, bool pdl) {
    const uint32_t groups = (n_tok + GROUP - 1) / GROUP;
    cudaError_t e = launch_kernel(delta_prep_kernel<2 * KP>, dim3((groups + 7) / 8, a.heads), dim3(256), 0, s, pdl, a, n_tok);
    if (e != cudaSuccess) return e;
    return 4u * KP * a.heads <= (uint32_t)sm_count ? scan_nc<KP, 2>(s, a, n_tok, pdl) : scan_nc<KP, 4>(s, a, n_tok, pdl);
}

}  // namespace

uint32_t delta_row(uint32_t dim) { return dim <= 256 ? (dim + 63u) & ~63u : 0u; }
size_t delta_record_floats(uint32_t n_tok, uint32_t heads, uint32_t drow) { return (size_t)((n_tok + GROUP - 1) / GROUP) * heads * group_floats(drow); }
bool delta_step_fits(const DeltaArgs &a) { return step_vec_smem(a.drow, (a.rank + 63) / 64 * 64) <= 200 * 1024; }

template <bool F32, bool STAGED> static cudaError_t step_launch(cudaStream_t s, const DeltaArgs &a, size_t vec, size_t smem, bool pdl) {
    const uint32_t cs = a.drow / ST_COLS;
    auto k = a.drow == 64 ? delta_step_kernel<F32, 2, STAGED> : a.drow == 128 ? delta_step_kernel<F32, 4, STAGED> : a.drow == 192 ? delta_step_kernel<F32, 6, STAGED> : delta_step_kernel<F32, 8, STAGED>;
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(k), smem);
    return e != cudaSuccess ? e : launch_cluster(k, dim3(cs * a.heads), dim3(ST_THREADS), smem, s, pdl, cs, a, (uint32_t)vec);
}
cudaError_t launch_delta_step(cudaStream_t s, bool f32, const DeltaArgs &a, bool pdl) {
    const size_t vec = step_vec_smem(a.drow, (a.rank + 63) / 64 * 64), all = vec + (size_t)(a.dim + 8) * 128 * a.decay.panels;
    return f32 ? step_launch<true, false>(s, a, vec, vec, pdl) : all <= 200 * 1024 ? step_launch<false, true>(s, a, vec, all, pdl) : step_launch<false, false>(s, a, vec, vec, pdl);
}
cudaError_t launch_delta_tanh(cudaStream_t s, bool f32, const DeltaArgs &a, const Act &out, uint32_t n_tok, bool pdl) {
    return launch_kernel(f32 ? delta_tanh_kernel<true> : delta_tanh_kernel<false>, dim3((n_tok * a.rank + 255) / 256), dim3(256), 0, s, pdl,
                         a.in + (size_t)5 * a.heads * a.dim, a.in_stride, a.rank, n_tok, out);
}
cudaError_t launch_delta_prompt(cudaStream_t s, bool f32, const DeltaArgs &a, uint32_t n_tok, int sm_count, bool pdl) {
    const dim3 grid((n_tok + 7) / 8, a.heads);
    cudaError_t e = cudaErrorInvalidValue;
    switch (a.drow / 64) {
        case 1: e = scan_kp<1>(s, a, n_tok, sm_count, pdl); break;
        case 2: e = scan_kp<2>(s, a, n_tok, sm_count, pdl); break;
        case 3: e = scan_kp<3>(s, a, n_tok, sm_count, pdl); break;
        case 4: e = scan_kp<4>(s, a, n_tok, sm_count, pdl); break;
        default: break;
    }
    if (e != cudaSuccess) return e;
    return launch_kernel(f32 ? delta_post_kernel<true> : delta_post_kernel<false>, grid, dim3(256), 0, s, pdl, a, n_tok);
}

}  // namespace k2t
