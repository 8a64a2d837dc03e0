// Sliding-window attention of the block engine (k2t_block_kernels.h): grouped queries, per-head score scale, a linear distance
// bias per head, unquantized (bf16 or fp32) key and value rows in a ring per layer.
//   * window_prep_kernel: per-head RMS norm of queries and keys of a prompt batch, cache rows, query rows (one warp per head).
//   * window_flash_kernel (bf16 prompts): CTA = 128 query rows of one kv head - row = (token, head of the group), so all heads
//     of a group share the key and value tiles - against 64-position tiles of the window, double-buffered with cp.async; both
//     products on the tensor cores (bf16 operands, fp32 accumulators), scores, bias, online softmax and its sums in fp32.
//   * window_row_kernel: one token and kv head per thread-block cluster.  The positions are split over the CTAs of the cluster,
//     partial maxima, sums and outputs are merged through distributed shared memory, so a decode step is ONE launch: norms of
//     the new query and key, the new cache row, attention and the activation of the output projection.  With fp32 rows the same
//     kernel serves prompts (grid.z = token).
#include <algorithm>

#include "k2t_block_kernels.h"
#include "k2t_dense.cuh"

namespace k2t {
namespace {

constexpr uint32_t ROW_MAX = 256;
constexpr float LOG2E = 1.4426950408889634f;

template <typename T> __device__ __forceinline__ void put(T *p, float v);
template <> __device__ __forceinline__ void put<float>(float *p, float v) { *p = v; }
template <> __device__ __forceinline__ void put<__nv_bfloat16>(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }

// eight consecutive elements of a cached row (plain loads: the row may have been written by this CTA)
__device__ __forceinline__ void get8(const float *p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4 *>(p), b = *reinterpret_cast<const float4 *>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void get8(const __nv_bfloat16 *p, float (&v)[8]) {
    const uint4 a = *reinterpret_cast<const uint4 *>(p);
    v[0] = bf_lo(a.x); v[1] = bf_hi(a.x); v[2] = bf_lo(a.y); v[3] = bf_hi(a.y); v[4] = bf_lo(a.z); v[5] = bf_hi(a.z); v[6] = bf_lo(a.w); v[7] = bf_hi(a.w);
}

// one warp: dst[0 .. row) = x / rms(x) * w for dim values, zeros behind
template <typename T> __device__ __forceinline__ void norm_row(const float *x, const float *w, uint32_t dim, uint32_t row, float eps, T *dst, uint32_t lane) {
    float v[ROW_MAX / 32], ss = 0.0f;
#pragma unroll
    for (uint32_t i = 0; i < ROW_MAX / 32; ++i) {
        const uint32_t k = lane + 32 * i;
        v[i] = k < dim ? __ldcg(x + k) : 0.0f;
        ss = __fmaf_rn(v[i], v[i], ss);
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
#pragma unroll
    for (uint32_t i = 0; i < ROW_MAX / 32; ++i) {
        const uint32_t k = lane + 32 * i;
        if (k < row) put<T>(dst + k, k < dim ? v[i] * inv * __ldg(w + k) : 0.0f);
    }
}
template <typename T> __device__ __forceinline__ void copy_row(const float *x, uint32_t dim, uint32_t row, T *dst, uint32_t lane) {
    for (uint32_t k = lane; k < row; k += 32) put<T>(dst + k, k < dim ? __ldcg(x + k) : 0.0f);
}

struct AttnParams {
    WindowAttnArgs a;
    uint32_t n_tok, ring_rows, fused;       // ring_rows = cache rows per kv head
};

template <typename T>
__global__ void __launch_bounds__(256) window_prep_kernel(const AttnParams p) {
    const WindowAttnArgs &a = p.a;
    const uint32_t lane = threadIdx.x & 31, heads = a.n_q + 2 * a.n_kv, t = blockIdx.y, h = blockIdx.x * 8 + (threadIdx.x >> 5);
    pdl_wait();
    pdl_trigger();
    if (h >= heads) return;
    const float *x = a.qkv + t * a.qkv_stride;
    const uint32_t slot = a.ring.slot_of_pos(__ldcg(a.pos) + t);
    if (h < a.n_q) {
        norm_row<T>(x + h * a.dim, a.q_norm, a.dim, a.row, a.eps, static_cast<T *>(a.q) + ((size_t)t * a.n_q + h) * a.row, lane);
    } else if (h < a.n_q + a.n_kv) {
        const uint32_t g = h - a.n_q;
        norm_row<T>(x + (a.n_q + g) * a.dim, a.k_norm, a.dim, a.row, a.eps, static_cast<T *>(a.k_cache) + ((size_t)g * p.ring_rows + slot) * a.row, lane);
    } else {
        const uint32_t g = h - a.n_q - a.n_kv;
        copy_row<T>(x + (a.n_q + a.n_kv) * a.dim + g * a.vdim, a.vdim, a.row, static_cast<T *>(a.v_cache) + ((size_t)g * p.ring_rows + slot) * a.row, lane);
    }
}

// ------------------------------------------------------------------------------------------------ one token per cluster
constexpr uint32_t RW_THREADS = 256, RW_SC = 256, RW_HB = 8, RW_PB = 4;
inline size_t rw_smem(uint32_t group, uint32_t row) { return ((size_t)group * (2 * row + RW_SC + 4) + 8 * RW_THREADS) * 4; }

template <typename T, int D>
__global__ void __launch_bounds__(RW_THREADS) window_row_kernel(const AttnParams p) {
    extern __shared__ __align__(16) float sm[];
    const WindowAttnArgs &a = p.a;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, cs = cluster_size(), me = cluster_rank();
    const uint32_t g = blockIdx.y, t = blockIdx.z, group = a.n_q / a.n_kv;
    float *s_q = sm, *s_o = s_q + group * D, *s_p = s_o + group * D, *s_m = s_p + group * RW_SC, *s_l = s_m + group, *s_al = s_l + group, *s_red = s_al + 2 * group;
    pdl_wait();
    pdl_trigger();
    const uint32_t pos = __ldcg(a.pos) + t;
    const uint32_t n_seen = a.ring.active_len(pos + 1), lo = pos + 1 - n_seen;          // sinks are 0: the seen positions are consecutive
    const uint32_t per = (n_seen + cs - 1) / cs, j_lo = lo + min(n_seen, me * per), j_hi = lo + min(n_seen, (me + 1) * per);
    T *kc = static_cast<T *>(a.k_cache) + (size_t)g * p.ring_rows * D, *vc = static_cast<T *>(a.v_cache) + (size_t)g * p.ring_rows * D;
    if (p.fused) {
        const float *x = a.qkv + t * a.qkv_stride;
        for (uint32_t h = warp; h < group; h += RW_THREADS / 32) norm_row<float>(x + (g * group + h) * a.dim, a.q_norm, a.dim, D, a.eps, s_q + h * D, lane);
        if (pos >= j_lo && pos < j_hi) {            // the CTA that attends to the new position stores its rows
            const uint32_t slot = a.ring.slot_of_pos(pos);
            if (warp == 7) norm_row<T>(x + (a.n_q + g) * a.dim, a.k_norm, a.dim, D, a.eps, kc + (size_t)slot * D, lane);
            if (warp == 6) copy_row<T>(x + (a.n_q + a.n_kv) * a.dim + g * a.vdim, a.vdim, D, vc + (size_t)slot * D, lane);
        }
    } else {
        const T *qr = static_cast<const T *>(a.q) + ((size_t)t * a.n_q + g * group) * D;
        for (uint32_t i = tid * 8; i < group * D; i += RW_THREADS * 8) {
            float v[8];
            get8(qr + i, v);
#pragma unroll
            for (int k = 0; k < 8; ++k) s_q[i + k] = v[k];
        }
    }
    for (uint32_t i = tid; i < group * D; i += RW_THREADS) s_o[i] = 0.0f;
    for (uint32_t i = tid; i < group; i += RW_THREADS) { s_m[i] = -INFINITY; s_l[i] = 0.0f; }
    __syncthreads();
    for (uint32_t j0 = j_lo; j0 < j_hi; j0 += RW_SC) {
        const uint32_t n = min(RW_SC, j_hi - j0);
        // scores: four lanes per key, sixteen keys per warp and step
        const uint32_t sub = lane & 3u, ki = lane >> 2;
        for (uint32_t b = warp * 16; b < n; b += RW_THREADS / 2) {
            const uint32_t ja = b + ki, jb = b + 8 + ki;
            const T *ka = kc + (size_t)a.ring.slot_of_pos(j0 + min(ja, n - 1)) * D, *kb = kc + (size_t)a.ring.slot_of_pos(j0 + min(jb, n - 1)) * D;
            for (uint32_t h0 = 0; h0 < group; h0 += RW_HB) {
                float da[RW_HB], db[RW_HB];
#pragma unroll
                for (uint32_t h = 0; h < RW_HB; ++h) da[h] = db[h] = 0.0f;
#pragma unroll
                for (uint32_t c = 0; c < D / 32; ++c) {
                    float va[8], vb[8];
                    const uint32_t k = (c * 4 + sub) * 8;
                    get8(ka + k, va);
                    get8(kb + k, vb);
#pragma unroll
                    for (uint32_t h = 0; h < RW_HB; ++h) {
                        if (h0 + h >= group) break;
                        const float4 q0 = *reinterpret_cast<const float4 *>(s_q + (h0 + h) * D + k), q1 = *reinterpret_cast<const float4 *>(s_q + (h0 + h) * D + k + 4);
                        const float q[8] = {q0.x, q0.y, q0.z, q0.w, q1.x, q1.y, q1.z, q1.w};
#pragma unroll
                        for (int i = 0; i < 8; ++i) { da[h] = __fmaf_rn(q[i], va[i], da[h]); db[h] = __fmaf_rn(q[i], vb[i], db[h]); }
                    }
                }
#pragma unroll
                for (uint32_t h = 0; h < RW_HB; ++h) {
                    if (h0 + h >= group) break;
                    float u = da[h], w = db[h];
                    u = __fadd_rn(u, __shfl_xor_sync(0xffffffffu, u, 1)); w = __fadd_rn(w, __shfl_xor_sync(0xffffffffu, w, 1));
                    u = __fadd_rn(u, __shfl_xor_sync(0xffffffffu, u, 2)); w = __fadd_rn(w, __shfl_xor_sync(0xffffffffu, w, 2));
                    if (sub == (h & 3u)) {
                        const uint32_t hh = g * group + h0 + h;
                        const float sc = __ldg(a.head_scale + hh), sl = __ldg(a.head_slope + hh);
                        if (ja < n) s_p[(h0 + h) * RW_SC + ja] = u * sc - sl * (float)(pos - (j0 + ja));
                        if (jb < n) s_p[(h0 + h) * RW_SC + jb] = w * sc - sl * (float)(pos - (j0 + jb));
                    }
                }
            }
        }
        __syncthreads();
        for (uint32_t h = warp; h < group; h += RW_THREADS / 32) {          // softmax terms of the tile, one warp per head
            float mx = -INFINITY;
            for (uint32_t j = lane; j < n; j += 32) mx = fmaxf(mx, s_p[h * RW_SC + j]);
#pragma unroll
            for (int m = 16; m > 0; m >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, m));
            const float m_old = s_m[h], m_new = fmaxf(m_old, mx);
            float sum = 0.0f;
            for (uint32_t j = lane; j < n; j += 32) { const float e = expf(s_p[h * RW_SC + j] - m_new); s_p[h * RW_SC + j] = e; sum += e; }
            sum = warp_sum(sum);
            if (lane == 0) { const float al = expf(m_old - m_new); s_al[h] = al; s_m[h] = m_new; s_l[h] = s_l[h] * al + sum; }
        }
        __syncthreads();
        // values: thread = (key slice, eight columns)
        constexpr uint32_t CPK = D / 8, KS = RW_THREADS / CPK;
        const uint32_t ks = tid / CPK, c = tid % CPK;
        for (uint32_t h0 = 0; h0 < group; h0 += RW_PB) {
            float acc[RW_PB][8];
#pragma unroll
            for (uint32_t h = 0; h < RW_PB; ++h)
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[h][i] = 0.0f;
            if (ks < KS)
#pragma unroll 4
                for (uint32_t j = ks; j < n; j += KS) {
                    float v[8];
                    get8(vc + (size_t)a.ring.slot_of_pos(j0 + j) * D + c * 8, v);
#pragma unroll
                    for (uint32_t h = 0; h < RW_PB; ++h) {
                        if (h0 + h >= group) break;
                        const float e = s_p[(h0 + h) * RW_SC + j];
#pragma unroll
                        for (int i = 0; i < 8; ++i) acc[h][i] = __fmaf_rn(e, v[i], acc[h][i]);
                    }
                }
#pragma unroll
            for (uint32_t h = 0; h < RW_PB; ++h) {
                if (h0 + h >= group) break;
                if (ks < KS)
#pragma unroll
                    for (int i = 0; i < 8; ++i) s_red[ks * D + c * 8 + i] = acc[h][i];
                __syncthreads();
                for (uint32_t d = tid; d < D; d += RW_THREADS) {
                    float o = 0.0f;
                    for (uint32_t k = 0; k < KS; ++k) o = __fadd_rn(o, s_red[k * D + d]);
                    s_o[(h0 + h) * D + d] = s_o[(h0 + h) * D + d] * s_al[h0 + h] + o;
                }
                __syncthreads();
            }
        }
    }
    // merge over the cluster: CTA r finishes the group's heads r, r + cs, ..
    if (cs > 1) cluster_sync_all();
    for (uint32_t h = me; h < group; h += cs) {
        float m = -INFINITY, l = 0.0f;
        for (uint32_t r = 0; r < cs; ++r) m = fmaxf(m, cs > 1 ? ld_cluster_f32(s_m + h, r) : s_m[h]);
        float f[16];
#pragma unroll
        for (uint32_t r = 0; r < 16; ++r) {
            f[r] = 0.0f;
            if (r < cs) {
                f[r] = expf((cs > 1 ? ld_cluster_f32(s_m + h, r) : s_m[h]) - m);
                l += f[r] * (cs > 1 ? ld_cluster_f32(s_l + h, r) : s_l[h]);
            }
        }
        const float inv = 1.0f / l;
        for (uint32_t d = tid; d < a.vdim; d += RW_THREADS) {
            float o = 0.0f;
#pragma unroll
            for (uint32_t r = 0; r < 16; ++r)
                if (r < cs) o = __fmaf_rn(f[r], cs > 1 ? ld_cluster_f32(s_o + h * D + d, r) : s_o[h * D + d], o);
            act_store<sizeof(T) == 4>(a.out, t, (g * group + h) * a.vdim + d, o * inv);
        }
    }
    if (cs > 1) cluster_sync_all();
}

// ------------------------------------------------------------------------------------------------ prompts, bf16
constexpr uint32_t FL_M = 128, FL_N = 64, FL_THREADS = 256;
__host__ __device__ constexpr uint32_t fl_pitch(uint32_t d) { return d * 2 + 16; }          // bytes; the pad spreads eight rows over all banks
__host__ __device__ constexpr uint32_t fl_smem(uint32_t d) { return fl_pitch(d) * (FL_M + 4 * FL_N); }

__device__ __forceinline__ void fl_cp16(uint32_t dst, const void *src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t &a, uint32_t &b, uint32_t &c, uint32_t &d) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(a), "=r"(b), "=r"(c), "=r"(d) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t &a, uint32_t &b, uint32_t &c, uint32_t &d) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(a), "=r"(b), "=r"(c), "=r"(d) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int D>
__global__ void __launch_bounds__(FL_THREADS) window_flash_kernel(const AttnParams p) {
    extern __shared__ __align__(16) uint8_t sm8[];
    const WindowAttnArgs &a = p.a;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = blockIdx.y, group = a.n_q / a.n_kv;
    const uint32_t rows = p.n_tok * group, r0 = blockIdx.x * FL_M;
    constexpr uint32_t P = fl_pitch(D), CH = D / 8;
    const uint32_t s_q = (uint32_t)__cvta_generic_to_shared(sm8), s_kv = s_q + FL_M * P;       // K0 | V0 | K1 | V1
    pdl_wait();
    pdl_trigger();
    const uint32_t pos0 = __ldcg(a.pos), r_last = min(rows, r0 + FL_M) - 1;
    const uint32_t p_first = pos0 + r0 / group, p_last = pos0 + r_last / group;
    const uint32_t lo = p_first + 1 - a.ring.active_len(p_first + 1);
    const __nv_bfloat16 *kc = static_cast<const __nv_bfloat16 *>(a.k_cache) + (size_t)g * p.ring_rows * D, *vc = static_cast<const __nv_bfloat16 *>(a.v_cache) + (size_t)g * p.ring_rows * D;
    for (uint32_t i = tid; i < FL_M * CH; i += FL_THREADS) {
        const uint32_t r = min(r0 + i / CH, rows - 1), c = i % CH;
        fl_cp16(s_q + (i / CH) * P + c * 16, static_cast<const __nv_bfloat16 *>(a.q) + ((size_t)(r / group) * a.n_q + g * group + r % group) * D + c * 8);
    }
    auto fetch = [&](uint32_t j0, uint32_t buf) {           // positions beyond the last are clamped (masked below, rows finite)
        for (uint32_t i = tid; i < FL_N * CH; i += FL_THREADS) {
            const uint32_t c = i % CH, slot = a.ring.slot_of_pos(min(j0 + i / CH, p_last));
            const uint32_t dst = s_kv + buf * 2 * FL_N * P + (i / CH) * P + c * 16;
            fl_cp16(dst, kc + (size_t)slot * D + c * 8);
            fl_cp16(dst + FL_N * P, vc + (size_t)slot * D + c * 8);
        }
    };
    fetch(lo, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    // the two query rows of this thread
    uint32_t qpos[2];
    float sc[2], sl[2], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const uint32_t r = min(r0 + warp * 16 + (lane >> 2) + 8 * i, rows - 1);
        qpos[i] = pos0 + r / group;
        sc[i] = __ldg(a.head_scale + g * group + r % group) * LOG2E;
        sl[i] = __ldg(a.head_slope + g * group + r % group) * LOG2E;
    }
    const uint32_t window = a.ring.window ? a.ring.window : 0xffffffffu;
    // positions some row of this warp can see
    const uint32_t w_first = pos0 + min(r0 + warp * 16, rows - 1) / group, w_last = pos0 + min(r0 + warp * 16 + 15, rows - 1) / group;
    const uint32_t w_lo = w_first + 1 - a.ring.active_len(w_first + 1);
    float o[D / 8][4];
#pragma unroll
    for (int i = 0; i < D / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    uint32_t buf = 0;
    for (uint32_t j0 = lo; j0 <= p_last; j0 += FL_N, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                     // the tile has landed; everyone is done with the other buffer
        if (j0 + FL_N <= p_last) fetch(j0 + FL_N, buf ^ 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (j0 > w_last || j0 + FL_N <= w_lo) continue;
        const uint32_t s_k = s_kv + buf * 2 * FL_N * P, s_v = s_k + FL_N * P;
        float s[FL_N / 8][4];
#pragma unroll
        for (int i = 0; i < (int)FL_N / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
#pragma unroll
        for (uint32_t k = 0; k < D / 16; ++k) {
            uint32_t a0, a1, a2, a3;
            ldsm4(s_q + (warp * 16 + (lane & 15u)) * P + k * 32 + (lane >> 4) * 16, a0, a1, a2, a3);
#pragma unroll
            for (uint32_t n = 0; n < FL_N / 16; ++n) {
                uint32_t b0, b1, b2, b3;       // keys n*16 .. +7 (k halves b0, b1), +8 .. +15 (b2, b3)
                ldsm4(s_k + (n * 16 + (lane & 7u) + ((lane >> 4) << 3)) * P + k * 32 + ((lane >> 3) & 1u) * 16, b0, b1, b2, b3);
                mma_bf16(s[2 * n], a0, a1, a2, a3, b0, b1);
                mma_bf16(s[2 * n + 1], a0, a1, a2, a3, b2, b3);
            }
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (uint32_t n = 0; n < FL_N / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t i = e >> 1, j = j0 + n * 8 + (lane & 3u) * 2 + (e & 1);
                const uint32_t dist = qpos[i] - j;            // wraps for later positions: larger than any window
                const bool seen = j <= qpos[i] && dist < window;
                const float v = seen ? __fmaf_rn(s[n][e], sc[i], -sl[i] * (float)dist) : -INFINITY;
                s[n][e] = v;
                mx[i] = fmaxf(mx[i], v);
            }
        float al[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
            const float m_new = fmaxf(m[i], mx[i]);
            al[i] = m_new == -INFINITY ? 1.0f : exp2f(m[i] - m_new);
            m[i] = m_new;
            l[i] *= al[i];
        }
#pragma unroll
        for (uint32_t n = 0; n < FL_N / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float mm = m[e >> 1];
                const float v = mm == -INFINITY ? 0.0f : exp2f(s[n][e] - mm);
                s[n][e] = v;
                l[e >> 1] += v;
            }
#pragma unroll
        for (int i = 0; i < D / 8; ++i) { o[i][0] *= al[0]; o[i][1] *= al[0]; o[i][2] *= al[1]; o[i][3] *= al[1]; }
#pragma unroll
        for (uint32_t k = 0; k < FL_N / 16; ++k) {
            const uint32_t a0 = pack_bf16(s[2 * k][0], s[2 * k][1]), a1 = pack_bf16(s[2 * k][2], s[2 * k][3]), a2 = pack_bf16(s[2 * k + 1][0], s[2 * k + 1][1]),
                           a3 = pack_bf16(s[2 * k + 1][2], s[2 * k + 1][3]);
#pragma unroll
            for (uint32_t d = 0; d < D / 16; ++d) {
                uint32_t b0, b1, b2, b3;
                ldsm4t(s_v + (k * 16 + (lane & 15u)) * P + d * 32 + (lane >> 4) * 16, b0, b1, b2, b3);
                mma_bf16(o[2 * d], a0, a1, a2, a3, b0, b1);
                mma_bf16(o[2 * d + 1], a0, a1, a2, a3, b2, b3);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
        const uint32_t r = r0 + warp * 16 + (lane >> 2) + 8 * i;
        if (r >= rows) continue;
        const float inv = 1.0f / l[i];
        const uint32_t t = r / group, base = (g * group + r % group) * a.vdim;
#pragma unroll
        for (int d = 0; d < D / 8; ++d) {
            const uint32_t k = d * 8 + (lane & 3u) * 2;
            if (k + 1 < a.vdim && (base & 1u) == 0)
                *reinterpret_cast<uint32_t *>(static_cast<__nv_bfloat16 *>(a.out.p) + panel_index(a.out.ld, t, base + k)) = pack_bf16(o[d][2 * i] * inv, o[d][2 * i + 1] * inv);
            else {
                if (k < a.vdim) act_store<false>(a.out, t, base + k, o[d][2 * i] * inv);
                if (k + 1 < a.vdim) act_store<false>(a.out, t, base + k + 1, o[d][2 * i + 1] * inv);
            }
        }
    }
}

template <typename T, int D>
cudaError_t row_launch(cudaStream_t s, const AttnParams &p, int sm_count, bool pdl) {
    const WindowAttnArgs &a = p.a;
    const uint32_t group = a.n_q / a.n_kv;
    uint32_t cs = 1;                            // CTAs per (token, kv head): at least 64 positions each, about one wave of CTAs
    const uint32_t longest = a.ring.window ? a.ring.window : p.ring_rows;
    while (cs < 8 && cs * 2 * 64 <= longest && cs * 2 * a.n_kv * p.n_tok <= (uint32_t)sm_count) cs *= 2;
    const size_t smem = rw_smem(group, D);
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(window_row_kernel<T, D>), smem);
    if (e != cudaSuccess) return e;
    return launch_cluster(window_row_kernel<T, D>, dim3(cs, a.n_kv, p.n_tok), dim3(RW_THREADS), smem, s, pdl, cs, p);
}
template <int D>
cudaError_t flash_launch(cudaStream_t s, const AttnParams &p, bool pdl) {
    const uint32_t rows = p.n_tok * (p.a.n_q / p.a.n_kv);
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(window_flash_kernel<D>), fl_smem(D));
    if (e != cudaSuccess) return e;
    return launch_kernel(window_flash_kernel<D>, dim3((rows + FL_M - 1) / FL_M, p.a.n_kv), dim3(FL_THREADS), fl_smem(D), s, pdl, p);
}

}  // namespace

uint32_t window_attn_row(uint32_t dim, uint32_t vdim) {
    const uint32_t d = std::max(dim, vdim);
    for (uint32_t c : {32u, 64u, 96u, 128u, 192u, 256u})
        if (d <= c) return c;
    return 0;
}

cudaError_t launch_window_attention(cudaStream_t s, bool f32, const WindowAttnArgs &a, uint32_t n_tok, int sm_count, uint32_t *launches, bool pdl) {
    AttnParams p{a, n_tok, 0, n_tok == 1 ? 1u : 0u};
    p.ring_rows = a.ring.ring_len;
    if (n_tok > 65535u || rw_smem(a.n_q / a.n_kv, a.row) > 220 * 1024) return cudaErrorInvalidValue;
    *launches = n_tok == 1 ? 1 : 2;
    if (n_tok > 1) {
        const dim3 grid((a.n_q + 2 * a.n_kv + 7) / 8, n_tok);
        cudaError_t e = f32 ? launch_kernel(window_prep_kernel<float>, grid, dim3(256), 0, s, pdl, p) : launch_kernel(window_prep_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl, p);
        if (e != cudaSuccess) return e;
    }
#define K2T_ROW(D) case D: return f32 ? row_launch<float, D>(s, p, sm_count, pdl) : n_tok == 1 ? row_launch<__nv_bfloat16, D>(s, p, sm_count, pdl) : flash_launch<D>(s, p, pdl)
    switch (a.row) {
        K2T_ROW(32);
        K2T_ROW(64);
        K2T_ROW(96);
        K2T_ROW(128);
        K2T_ROW(192);
        K2T_ROW(256);
        default: return cudaErrorInvalidValue;
    }
#undef K2T_ROW
}

}  // namespace k2t
