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
// The heads of a group run in passes of HB (the group is padded to full passes with zero queries), so the inner loops carry no
// branches.  Cached rows come in tiles by bulk copy (a CTA's positions are consecutive, so a tile is one run of the ring, two
// where it wraps); a decode step asks for its first tiles before its dependency wait - earlier steps wrote those rows - and lays
// the new position's row over the stale one once the tile has landed.
constexpr uint32_t RW_THREADS = 256, RW_MAX_CS = 8;
constexpr uint32_t RW_WAIT_LIMIT = 1u << 22;
// positions per tile: 64 KiB of keys (32 for long passes and fp32 rows), at most 256, a multiple of 16
template <typename T> __host__ __device__ constexpr uint32_t rw_tile(uint32_t row, uint32_t hb) {
    const uint32_t n = (hb > 4 || sizeof(T) == 4 ? 32768u : 65536u) / (row * (uint32_t)sizeof(T));
    return (n > 256u ? 256u : n) & ~15u;
}
__host__ __device__ inline uint32_t rw_pad(uint32_t group, uint32_t hb) { return (group + hb - 1) / hb * hb; }
template <typename T> inline size_t rw_smem(uint32_t group, uint32_t row, uint32_t hb) {
    const uint32_t tile = rw_tile<T>(row, hb);
    return (size_t)2 * tile * row * sizeof(T) + ((size_t)rw_pad(group, hb) * (2 * row + tile + 4 + 2 * RW_MAX_CS) + (size_t)8 * RW_THREADS * hb + 2 * row) * 4;
}

template <typename T, int D, int HB>
__global__ void __launch_bounds__(RW_THREADS) window_row_kernel(const AttnParams p) {
    extern __shared__ __align__(128) uint8_t smb[];
    __shared__ __align__(8) uint64_t bars[2];
    constexpr uint32_t TILE = rw_tile<T>(D, HB);
    const WindowAttnArgs &a = p.a;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, cs = cluster_size(), me = cluster_rank();
    const uint32_t g = blockIdx.y, t = blockIdx.z, group = a.n_q / a.n_kv, gp = rw_pad(group, HB);
    T *s_k = reinterpret_cast<T *>(smb), *s_v = s_k + TILE * D;
    float *s_q = reinterpret_cast<float *>(s_v + TILE * D), *s_o = s_q + gp * D, *s_red = s_o + gp * D, *s_new = s_red + 8 * RW_THREADS * HB, *s_p = s_new + 2 * D, *s_m = s_p + gp * TILE,
          *s_l = s_m + gp, *s_al = s_l + gp, *s_fm = s_al + 2 * gp, *s_fl = s_fm + gp * RW_MAX_CS;
    T *kc = static_cast<T *>(a.k_cache) + (size_t)g * p.ring_rows * D, *vc = static_cast<T *>(a.v_cache) + (size_t)g * p.ring_rows * D;
    const uint32_t bar = (uint32_t)__cvta_generic_to_shared(bars), sk = (uint32_t)__cvta_generic_to_shared(s_k), sv = (uint32_t)__cvta_generic_to_shared(s_v);
    if (tid == 0) { mbar_init(bar, 1); mbar_init(bar + 8, 1); fence_mbar_init(); }
    if (!p.fused) { pdl_wait(); pdl_trigger(); }
    const uint32_t pos = __ldcg(a.pos) + t;                                              // a decode step's position was set before the step began
    const uint32_t n_seen = a.ring.active_len(pos + 1), lo = pos + 1 - n_seen;          // sinks are 0: the seen positions are consecutive
    const uint32_t per = (n_seen + cs - 1) / cs, j_lo = lo + min(n_seen, me * per), j_hi = lo + min(n_seen, (me + 1) * per);
    // rows of positions j0 .. of one tile; a stale row of the new position may come along
    auto request = [&](uint32_t dst, const T *cache, uint32_t j0, uint32_t b) {
        const uint32_t n = min(TILE, j_hi - j0), slot = a.ring.slot_of_pos(j0), first = min(n, p.ring_rows - slot);
        mbar_expect_tx(b, n * D * (uint32_t)sizeof(T));
        bulk_g2s(dst, cache + (size_t)slot * D, first * D * (uint32_t)sizeof(T), b);
        if (first < n) bulk_g2s(dst + first * D * (uint32_t)sizeof(T), cache, (n - first) * D * (uint32_t)sizeof(T), b);
    };
    auto landed = [&](uint32_t b, uint32_t parity) {
        bool ok = false;
        for (uint32_t spin = 0; spin < RW_WAIT_LIMIT && !ok; ++spin) ok = mbar_try_wait(b, parity);
        if (!ok && a.err_flag != nullptr) atomicExch(a.err_flag, 1u);
    };
    if (tid == 0 && j_lo < j_hi) { request(sk, kc, j_lo, bar); request(sv, vc, j_lo, bar + 8); }
    for (uint32_t i = tid; i < gp * D; i += RW_THREADS) s_o[i] = 0.0f;
    for (uint32_t i = group * D + tid; i < gp * D; i += RW_THREADS) s_q[i] = 0.0f;
    for (uint32_t i = tid; i < gp; i += RW_THREADS) { s_m[i] = -INFINITY; s_l[i] = 0.0f; s_al[i] = 0.0f; }
    const bool owner = p.fused && pos >= j_lo && pos < j_hi;          // this CTA attends to the new position and stores its rows
    if (p.fused) {
        pdl_wait();
        pdl_trigger();
        const float *x = a.qkv + t * a.qkv_stride;
        for (uint32_t h = warp; h < group + (owner ? 2u : 0u); h += RW_THREADS / 32) {
            if (h < group) norm_row<float>(x + (g * group + h) * a.dim, a.q_norm, a.dim, D, a.eps, s_q + h * D, lane);
            else if (h == group) norm_row<float>(x + (a.n_q + g) * a.dim, a.k_norm, a.dim, D, a.eps, s_new, lane);
            else copy_row<float>(x + (a.n_q + a.n_kv) * a.dim + g * a.vdim, a.vdim, D, s_new + D, lane);
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
    __syncthreads();
    if (owner) {
        const size_t slot = (size_t)a.ring.slot_of_pos(pos) * D;
        for (uint32_t i = tid; i < D; i += RW_THREADS) { put<T>(kc + slot + i, s_new[i]); put<T>(vc + slot + i, s_new[D + i]); }
    }
    uint32_t phase = 0;
    for (uint32_t j0 = j_lo; j0 < j_hi; j0 += TILE, phase ^= 1) {
        const uint32_t n = min(TILE, j_hi - j0), j_next = j0 + TILE;
        const bool patch = owner && pos >= j0 && pos < j0 + n;
        landed(bar, phase);
        if (patch) {
            for (uint32_t i = tid; i < D; i += RW_THREADS) put<T>(s_k + (pos - j0) * D + i, s_new[i]);
            __syncthreads();
        }
        // scores: four lanes per key, sixteen keys per warp and step; neighbouring keys take their 64-byte pieces in another
        // order, so that the eight lanes of a shared-memory phase hit different banks
        const uint32_t sub = lane & 3u, ki = lane >> 2;
#pragma unroll 1
        for (uint32_t b = warp * 16; b < n; b += RW_THREADS / 2) {
            const uint32_t ja = b + ki, jb = b + 8 + ki;
            const T *ka = s_k + min(ja, n - 1) * D, *kb = s_k + min(jb, n - 1) * D;
#pragma unroll 1
            for (uint32_t h0 = 0; h0 < group; h0 += HB) {
                float da[HB], db[HB];
#pragma unroll
                for (uint32_t h = 0; h < HB; ++h) da[h] = db[h] = 0.0f;
#pragma unroll 1
                for (uint32_t c = 0; c < D / 32; ++c) {          // rolled: instruction fetch costs more than the loop
                    float va[8], vb[8];
                    const uint32_t k = (((c + (ki & 1u)) % (D / 32)) * 4 + sub) * 8;
                    get8(ka + k, va);
                    get8(kb + k, vb);
#pragma unroll
                    for (uint32_t h = 0; h < HB; ++h) {
                        const float4 q0 = *reinterpret_cast<const float4 *>(s_q + (h0 + h) * D + k), q1 = *reinterpret_cast<const float4 *>(s_q + (h0 + h) * D + k + 4);
                        const float q[8] = {q0.x, q0.y, q0.z, q0.w, q1.x, q1.y, q1.z, q1.w};
#pragma unroll
                        for (int i = 0; i < 8; ++i) { da[h] = __fmaf_rn(q[i], va[i], da[h]); db[h] = __fmaf_rn(q[i], vb[i], db[h]); }
                    }
                }
#pragma unroll
                for (int m = 1; m < 4; m <<= 1)
#pragma unroll
                    for (uint32_t h = 0; h < HB; ++h) {
                        da[h] = __fadd_rn(da[h], __shfl_xor_sync(0xffffffffu, da[h], m));
                        db[h] = __fadd_rn(db[h], __shfl_xor_sync(0xffffffffu, db[h], m));
                    }
#pragma unroll
                for (uint32_t h = 0; h < HB; ++h)
                    if (sub == (h & 3u)) {
                        const uint32_t hh = g * group + min(h0 + h, group - 1);
                        const float sc = __ldg(a.head_scale + hh), sl = __ldg(a.head_slope + hh);
                        if (ja < n) s_p[(h0 + h) * TILE + ja] = da[h] * sc - sl * (float)(pos - (j0 + ja));
                        if (jb < n) s_p[(h0 + h) * TILE + jb] = db[h] * sc - sl * (float)(pos - (j0 + jb));
                    }
            }
        }
        __syncthreads();
        if (tid == 0 && j_next < j_hi) request(sk, kc, j_next, bar);         // everyone is done with the keys
#pragma unroll 1
        for (uint32_t h = warp; h < group; h += RW_THREADS / 32) {          // softmax terms of the tile, one warp per head
            float mx = -INFINITY;
            for (uint32_t j = lane; j < n; j += 32) mx = fmaxf(mx, s_p[h * TILE + j]);
#pragma unroll
            for (int m = 16; m > 0; m >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, m));
            const float m_old = s_m[h], m_new = fmaxf(m_old, mx);
            float sum = 0.0f;
            for (uint32_t j = lane; j < n; j += 32) { const float e = expf(s_p[h * TILE + j] - m_new); s_p[h * TILE + j] = e; sum += e; }
            sum = warp_sum(sum);
            if (lane == 0) { const float al = expf(m_old - m_new); s_al[h] = al; s_m[h] = m_new; s_l[h] = s_l[h] * al + sum; }
        }
        landed(bar + 8, phase);
        if (patch)
            for (uint32_t i = tid; i < D; i += RW_THREADS) put<T>(s_v + (pos - j0) * D + i, s_new[D + i]);
        __syncthreads();
        // values: thread = (key slice, eight columns); padding heads multiply finite leftovers that nobody reads
        constexpr uint32_t CPK = D / 8, KS = RW_THREADS / CPK;
        const uint32_t ks = tid / CPK, c = tid % CPK;
#pragma unroll 1
        for (uint32_t h0 = 0; h0 < group; h0 += HB) {
            float acc[HB][8];
#pragma unroll
            for (uint32_t h = 0; h < HB; ++h)
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[h][i] = 0.0f;
            if (ks < KS) {
#pragma unroll 2
                for (uint32_t j = ks; j < n; j += KS) {
                    float v[8];
                    get8(s_v + j * D + c * 8, v);
#pragma unroll
                    for (uint32_t h = 0; h < HB; ++h) {
                        const float e = s_p[(h0 + h) * TILE + j];
#pragma unroll
                        for (int i = 0; i < 8; ++i) acc[h][i] = __fmaf_rn(e, v[i], acc[h][i]);
                    }
                }
#pragma unroll
                for (uint32_t h = 0; h < HB; ++h) {
                    float4 *dst = reinterpret_cast<float4 *>(s_red + (ks * HB + h) * D + c * 8);
                    dst[0] = make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]);
                    dst[1] = make_float4(acc[h][4], acc[h][5], acc[h][6], acc[h][7]);
                }
            }
            __syncthreads();
            for (uint32_t e = tid; e < HB * D; e += RW_THREADS) {
                float o = 0.0f;
#pragma unroll 8
                for (uint32_t k = 0; k < KS; ++k) o = __fadd_rn(o, s_red[k * HB * D + e]);
                s_o[h0 * D + e] = s_o[h0 * D + e] * s_al[h0 + e / D] + o;
            }
            __syncthreads();
        }
        if (tid == 0 && j_next < j_hi) request(sv, vc, j_next, bar + 8);     // everyone is done with the values
    }
    // merge over the cluster: factors of every (head, CTA), then the outputs shared out over all CTAs
    __syncthreads();
    if (cs > 1) cluster_sync_all();
    for (uint32_t i = tid; i < group * cs; i += RW_THREADS) {
        const uint32_t h = i / cs, r = i % cs;
        s_fm[h * RW_MAX_CS + r] = cs > 1 ? ld_cluster_f32(s_m + h, r) : s_m[h];
        s_fl[h * RW_MAX_CS + r] = cs > 1 ? ld_cluster_f32(s_l + h, r) : s_l[h];
    }
    __syncthreads();
    for (uint32_t h = tid; h < group; h += RW_THREADS) {
        float m = -INFINITY, l = 0.0f;
        for (uint32_t r = 0; r < cs; ++r) m = fmaxf(m, s_fm[h * RW_MAX_CS + r]);
        for (uint32_t r = 0; r < cs; ++r) { const float f = expf(s_fm[h * RW_MAX_CS + r] - m); s_fm[h * RW_MAX_CS + r] = f; l += f * s_fl[h * RW_MAX_CS + r]; }
        s_fl[h * RW_MAX_CS] = 1.0f / l;
    }
    __syncthreads();
    for (uint32_t e = me * RW_THREADS + tid; e < group * a.vdim; e += cs * RW_THREADS) {
        const uint32_t h = e / a.vdim, d = e % a.vdim;
        float o = 0.0f;
#pragma unroll
        for (uint32_t r = 0; r < RW_MAX_CS; ++r)
            if (r < cs) o = __fmaf_rn(s_fm[h * RW_MAX_CS + r], cs > 1 ? ld_cluster_f32(s_o + h * D + d, r) : s_o[h * D + d], o);
        act_store<sizeof(T) == 4>(a.out, t, (g * group + h) * a.vdim + d, o * s_fl[h * RW_MAX_CS]);
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

__device__ __forceinline__ float fl_exp2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

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
    const uint32_t window = a.ring.window ? a.ring.window : 0x7fffffffu;
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
        // bias of the tile's first key of this thread, the others follow in exact steps (small integers times the slope)
        const float f0[2] = {(float)(int)(j0 + (lane & 3u) * 2 - qpos[0]), (float)(int)(j0 + (lane & 3u) * 2 - qpos[1])};
#pragma unroll
        for (uint32_t n = 0; n < FL_N / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t i = e >> 1;
                s[n][e] = __fmaf_rn(s[n][e], sc[i], sl[i] * (f0[i] + (float)(n * 8 + (e & 1))));
            }
        if (j0 + FL_N - 1 > w_first || w_last >= j0 + window) {            // some key of the tile is out of some row's sight
#pragma unroll
            for (uint32_t n = 0; n < FL_N / 8; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const uint32_t i = e >> 1, j = j0 + n * 8 + (lane & 3u) * 2 + (e & 1);
                    if (j > qpos[i] || qpos[i] - j >= window) s[n][e] = -INFINITY;
                }
        }
#pragma unroll
        for (uint32_t n = 0; n < FL_N / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) mx[e >> 1] = fmaxf(mx[e >> 1], s[n][e]);
        float al[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
            const float m_new = fmaxf(m[i], mx[i]);
            al[i] = m_new == -INFINITY ? 1.0f : fl_exp2(m[i] - m_new);
            m[i] = m_new;
            l[i] *= al[i];
        }
        const float mm[2] = {m[0] == -INFINITY ? 0.0f : m[0], m[1] == -INFINITY ? 0.0f : m[1]};        // a row that has seen nothing yet: exp2(-inf) = 0
#pragma unroll
        for (uint32_t n = 0; n < FL_N / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float v = fl_exp2(s[n][e] - mm[e >> 1]);
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

template <typename T, int D, int HB>
cudaError_t row_launch_hb(cudaStream_t s, const AttnParams &p, int sm_count, bool pdl) {
    const WindowAttnArgs &a = p.a;
    uint32_t cs = 1;                            // CTAs per (token, kv head): at least 64 positions each, about one wave of CTAs
    const uint32_t longest = a.ring.window ? a.ring.window : p.ring_rows;
    while (cs < RW_MAX_CS && cs * 2 * 64 <= longest && cs * 2 * a.n_kv * p.n_tok <= (uint32_t)sm_count) cs *= 2;
    const size_t smem = rw_smem<T>(a.n_q / a.n_kv, D, HB);
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(window_row_kernel<T, D, HB>), smem);
    if (e != cudaSuccess) return e;
    return launch_cluster(window_row_kernel<T, D, HB>, dim3(cs, a.n_kv, p.n_tok), dim3(RW_THREADS), smem, s, pdl, cs, p);
}
inline uint32_t head_pass(bool f32, uint32_t group) { return f32 ? 4u : group == 1 ? 1u : group <= 4 ? 4u : 8u; }
template <int D>
cudaError_t row_launch(cudaStream_t s, bool f32, const AttnParams &p, int sm_count, bool pdl) {
    if (f32) return row_launch_hb<float, D, 4>(s, p, sm_count, pdl);
    switch (head_pass(false, p.a.n_q / p.a.n_kv)) {
        case 1: return row_launch_hb<__nv_bfloat16, D, 1>(s, p, sm_count, pdl);
        case 4: return row_launch_hb<__nv_bfloat16, D, 4>(s, p, sm_count, pdl);
        default: return row_launch_hb<__nv_bfloat16, D, 8>(s, p, sm_count, pdl);
    }
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

bool window_attn_fits(bool f32, uint32_t group, uint32_t row) { return (f32 ? rw_smem<float>(group, row, head_pass(f32, group)) : rw_smem<__nv_bfloat16>(group, row, head_pass(f32, group))) <= 224 * 1024; }

cudaError_t launch_window_attention(cudaStream_t s, bool f32, const WindowAttnArgs &a, uint32_t n_tok, int sm_count, uint32_t *launches, bool pdl) {
    AttnParams p{a, n_tok, 0, n_tok == 1 ? 1u : 0u};
    p.ring_rows = a.ring.ring_len;
    if (n_tok > 65535u || !window_attn_fits(f32, a.n_q / a.n_kv, a.row)) return cudaErrorInvalidValue;
    *launches = n_tok == 1 ? 1 : 2;
    if (n_tok > 1) {
        const dim3 grid((a.n_q + 2 * a.n_kv + 7) / 8, n_tok);
        cudaError_t e = f32 ? launch_kernel(window_prep_kernel<float>, grid, dim3(256), 0, s, pdl, p) : launch_kernel(window_prep_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl, p);
        if (e != cudaSuccess) return e;
    }
#define K2T_ROW(D) case D: return f32 || n_tok == 1 ? row_launch<D>(s, f32, p, sm_count, pdl) : flash_launch<D>(s, p, pdl)
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
