// Latent attention of the block engine (k2t_block_kernels.h): low-rank queries, and one cached row (c, k_rot) per position that all
// heads share.  bf16 rows lie in 64-column panels of `ld` positions (k2t_dense.h), so the cache is the operand of the expanding
// product, a tile of positions is one contiguous run per panel, and its 128-byte swizzle suits both kinds of tensor-core operand.
//   * latent_prep_kernel: norms of both latents, rotation of the shared key part, cache row.
//   * few tokens: latent_absorb_kernel (W_uk^T q, rotation), latent_split_kernel (rows = (token, head), 16 or 32 of them against
//     64-position tiles of one split of the positions, mma.sync, online softmax in fp32), latent_value_kernel (merge of the
//     splits, W_uv).  latent_split_f32_kernel is the fp32 form.
//   * prompt batches, bf16: latent_query_kernel (rotation, operand panels), latent_flash_kernel: 128 tokens of a head per CTA,
//     S = Q K^T and O += P V by tcgen05.mma with S, P and O in tensor memory; tiles by bulk copy, the next S is computed
//     while the softmax of this one runs, O is rescaled only when a row's maximum has grown by more than 2^8.
#include <algorithm>

#include "k2t_block_kernels.h"
#include "k2t_dense.cuh"

namespace k2t {
namespace {

constexpr float LOG2E = 1.4426950408889634f;
constexpr uint32_t WAIT_LIMIT = 1u << 22;

__device__ __forceinline__ float exp2_approx(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// ------------------------------------------------------------------------------------------------ latents, cache row
// grid (token, 2): the query latent; the cache row
constexpr uint32_t PREP_THREADS = 512;
template <bool F32>
__global__ void __launch_bounds__(PREP_THREADS) latent_prep_kernel(const LatentAttnArgs a) {
    __shared__ float scratch[32];
    const LatentShape &d = a.d;
    const uint32_t t = blockIdx.x, tid = threadIdx.x, step = blockDim.x, n = blockIdx.y == 0 ? d.q_rank : d.kv_rank;
    const float *w = blockIdx.y == 0 ? a.q_norm : a.kv_norm;
    pdl_wait();
    pdl_trigger();
    const float *x = a.in + t * a.in_stride + (blockIdx.y == 0 ? 0 : d.q_rank);
    const uint32_t pos = __ldcg(a.pos) + t;
    constexpr uint32_t KEEP = 4;               // the thread's first values stay in registers
    float keep[KEEP], ss[1] = {0.0f};
#pragma unroll
    for (uint32_t i = 0; i < KEEP; ++i) { const uint32_t k = tid + i * step; keep[i] = k < n ? __ldcg(x + k) : 0.0f; }
#pragma unroll
    for (uint32_t i = 0; i < KEEP; ++i) ss[0] = __fmaf_rn(keep[i], keep[i], ss[0]);
    for (uint32_t k = tid + KEEP * step; k < n; k += step) { const float v = __ldcg(x + k); ss[0] = __fmaf_rn(v, v, ss[0]); }
    block_sum<1>(ss, scratch);
    const float inv = 1.0f / sqrtf(ss[0] / (float)n + a.eps);
    const Act &out = blockIdx.y == 0 ? a.q_lat : a.cache;
    const uint32_t row = blockIdx.y == 0 ? t : pos;
#pragma unroll
    for (uint32_t i = 0; i < KEEP; ++i) { const uint32_t k = tid + i * step; if (k < n) act_store<F32>(out, row, k, keep[i] * inv * __ldg(w + k)); }
    for (uint32_t k = tid + KEEP * step; k < n; k += step) act_store<F32>(out, row, k, __ldcg(x + k) * inv * __ldg(w + k));
    if (blockIdx.y == 1)
        for (uint32_t i = tid; i < d.rot_dim / 2; i += step) {
            const float u = __ldcg(x + d.kv_rank + 2 * i), v = __ldcg(x + d.kv_rank + 2 * i + 1);
            const float c = __ldg(a.rot + (size_t)pos * d.rot_dim + 2 * i), s = __ldg(a.rot + (size_t)pos * d.rot_dim + 2 * i + 1);
            act_store<F32>(a.cache, pos, d.rot_at + 2 * i, u * c - v * s);
            act_store<F32>(a.cache, pos, d.rot_at + 2 * i + 1, v * c + u * s);
        }
}

__device__ __forceinline__ float rotated(const float *q, const float *cs, uint32_t i) {      // element i of the rotated vector
    const float u = __ldcg(q + (i & ~1u)), v = __ldcg(q + (i | 1u)), c = __ldg(cs + (i & ~1u)), s = __ldg(cs + (i | 1u));
    return (i & 1u) ? v * c + u * s : u * c - v * s;
}

// ------------------------------------------------------------------------------------------------ few tokens: queries
// grid (panels of the latent + 1, head, tokens / NT).  A warp reads four rows of W_uk at a time, lane = (row, eight columns).
template <int NT>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const LatentAttnArgs a, uint32_t t_first, uint32_t t_end) {
    __shared__ float s_q[NT][256 + 4], s_red[8][NT][64];
    const LatentShape &d = a.d;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, t0 = t_first + blockIdx.z * NT, nt = min((uint32_t)NT, t_end - t0);
    const uint32_t panel = blockIdx.x, panels = d.rot_at / PANEL, c = lane & 7u, r4 = lane >> 3, per = d.dim + d.rot_dim;
    constexpr uint32_t PF = 4;
    uint4 w[PF];
    const uint4 *base = static_cast<const uint4 *>(a.kv_up.base) + ((size_t)panel * a.kv_up.rows_pad + h * latent_head_cols(d.dim)) * 8;
    if (panel < panels)
#pragma unroll
        for (uint32_t i = 0; i < PF; ++i) {
            const uint32_t k = (i * 8 + warp) * 4 + r4;
            w[i] = k < d.dim ? ldg_stream(base + (size_t)k * 8 + (c ^ (k & 7u))) : make_uint4(0, 0, 0, 0);
        }
    pdl_wait();
    pdl_trigger();
    if (panel == panels) {              // rotated part and its padding
        const uint32_t n = d.row - d.rot_at, pos = __ldcg(a.pos);
        for (uint32_t i = tid; i < nt * n; i += 256) {
            const uint32_t t = t0 + i / n, k = i % n;
            act_store<false>(a.q_rows, (t - t_first) * d.heads + h, d.rot_at + k, k < d.rot_dim ? rotated(a.q + t * a.q_stride + h * per + d.dim, a.rot + (size_t)(pos + t) * d.rot_dim, k) : 0.0f);
        }
        return;
    }
    float acc[NT][8];
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[t][i] = 0.0f;
    for (uint32_t k0 = 0; k0 < d.dim; k0 += 256) {        // a stretch of up to 256 query elements
        __syncthreads();
        for (uint32_t i = tid; i < NT * 256; i += 256) {
            const uint32_t t = i >> 8, k = k0 + (i & 255u);
            s_q[t][i & 255u] = t < nt && k < d.dim ? __ldcg(a.q + (t0 + t) * a.q_stride + h * per + k) : 0.0f;
        }
        __syncthreads();
        for (uint32_t b = 0; b < 8; b += PF) {
#pragma unroll
            for (uint32_t i = 0; i < PF; ++i) {
                const uint32_t j = ((b + i) * 8 + warp) * 4 + r4, k = k0 + j;
                if (k0 + (b + i) * 32 >= d.dim) break;
                const uint4 v = w[i];
                const uint32_t kn = k + PF * 32;
                w[i] = kn < d.dim ? ldg_stream(base + (size_t)kn * 8 + (c ^ (kn & 7u))) : make_uint4(0, 0, 0, 0);
                const float f[8] = {bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y), bf_lo(v.z), bf_hi(v.z), bf_lo(v.w), bf_hi(v.w)};
#pragma unroll
                for (int t = 0; t < NT; ++t) {
                    const float q = s_q[t][j];
#pragma unroll
                    for (int e = 0; e < 8; ++e) acc[t][e] = __fmaf_rn(f[e], q, acc[t][e]);
                }
            }
        }
    }
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            acc[t][e] = __fadd_rn(acc[t][e], __shfl_xor_sync(0xffffffffu, acc[t][e], 8));
            acc[t][e] = __fadd_rn(acc[t][e], __shfl_xor_sync(0xffffffffu, acc[t][e], 16));
        }
    if (r4 == 0)
#pragma unroll
        for (int t = 0; t < NT; ++t)
#pragma unroll
            for (int e = 0; e < 8; ++e) s_red[warp][t][c * 8 + e] = acc[t][e];
    __syncthreads();
    for (uint32_t i = tid; i < nt * 64; i += 256) {
        const uint32_t t = i >> 6, k = i & 63u;
        float s = 0.0f;
#pragma unroll
        for (int v = 0; v < 8; ++v) s = __fadd_rn(s, s_red[v][t][k]);
        act_store<false>(a.q_rows, (t0 + t - t_first) * d.heads + h, panel * PANEL + k, s);
    }
}

__global__ void __launch_bounds__(256) latent_absorb_f32_kernel(const LatentAttnArgs a, uint32_t t_first) {
    const LatentShape &d = a.d;
    const uint32_t h = blockIdx.y, t = t_first + blockIdx.z, k = blockIdx.x * 256 + threadIdx.x, per = d.dim + d.rot_dim;
    pdl_wait();
    pdl_trigger();
    const float *q = a.q + t * a.q_stride + h * per;
    const uint32_t row = (t - t_first) * d.heads + h;
    if (k < d.kv_rank) {
        const float *w = static_cast<const float *>(a.kv_up.base) + (size_t)h * latent_head_cols(d.dim) * a.kv_up.rows_pad + k;
        float s = 0.0f;
        for (uint32_t i = 0; i < d.dim; ++i) s = __fmaf_rn(__ldg(w + (size_t)i * a.kv_up.rows_pad), __ldcg(q + i), s);
        act_store<true>(a.q_rows, row, k, s);
    } else if (k >= d.rot_at && k < d.rot_at + d.rot_dim) {
        act_store<true>(a.q_rows, row, k, rotated(q + d.dim, a.rot + (size_t)(__ldcg(a.pos) + t) * d.rot_dim, k - d.rot_at));
    }
}

// ------------------------------------------------------------------------------------------------ few tokens: cached rows
constexpr uint32_t SP_N = 64, SP_THREADS = 256;      // positions per tile
struct SplitParams {
    LatentAttnArgs a;
    uint32_t t0, rows, splits, stages;      // rows = tokens * heads
};
__host__ __device__ inline uint32_t part_stride(const LatentShape &d) { return (d.kv_rank + 3u) & ~3u; }
// tiles [first, last) of this split, of the tiles the launch's last token sees (alike for all rows: the merge counts on it)
__device__ __forceinline__ void split_range(uint32_t seen, uint32_t split, uint32_t splits, uint32_t &first, uint32_t &last) {
    const uint32_t tiles = (seen + SP_N - 1) / SP_N, per = (tiles + splits - 1) / splits;
    first = min(tiles, split * per);
    last = min(tiles, first + per);
}

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
// shared-memory address of 16-byte chunk `chunk` (of the whole row) of row `row` of a tile kept as panels of `rows` rows
__device__ __forceinline__ uint32_t tile_chunk(uint32_t base, uint32_t rows, uint32_t row, uint32_t chunk) {
    return base + (((chunk >> 3) * rows + row) * 8 + ((chunk & 7u) ^ (row & 7u))) * 16;
}

__host__ __device__ constexpr uint32_t sp_pitch() { return SP_N * 2 + 16; }          // bytes of a row of softmax weights
template <int RB> inline size_t sp_smem(const LatentShape &d, uint32_t stages) {
    return 128 + (size_t)d.row / PANEL * 128 * (16 * RB + stages * SP_N) + (size_t)16 * RB * ((SP_N + 4) * 4 + sp_pitch() + 3 * 4);
}

// CTA = 16 RB rows against one split.  Warp w: scores of keys 8 w .. 8 w + 7 of a tile; softmax of rows 2 RB w ..; values of
// the 16-column units w, w + 8, ... (U per warp) of the latent.
template <int RB, int U>
__global__ void __launch_bounds__(SP_THREADS) latent_split_kernel(const SplitParams p) {
    extern __shared__ __align__(128) uint8_t smb[];
    __shared__ __align__(8) uint64_t bars[3];
    constexpr uint32_t M = 16 * RB;
    const LatentAttnArgs &a = p.a;
    const LatentShape &d = a.d;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, r0 = blockIdx.y * M, n_row = min(M, p.rows - r0), split = blockIdx.x;
    const uint32_t panels = d.row / PANEL, raw = (uint32_t)__cvta_generic_to_shared(smb), base = (raw + 127u) & ~127u;
    const uint32_t s_q = base, s_t = s_q + panels * M * 128, tile_bytes = panels * SP_N * 128, s_p = s_t + p.stages * tile_bytes;
    uint8_t *gen = smb + (base - raw);
    float *s_s = reinterpret_cast<float *>(gen + (s_p - base) + M * sp_pitch()), *s_al = s_s + M * (SP_N + 4), *s_m = s_al + M, *s_l = s_m + M;
    __nv_bfloat16 *g_p = reinterpret_cast<__nv_bfloat16 *>(gen + (s_p - base));
    const uint32_t bar = (uint32_t)__cvta_generic_to_shared(bars);
    if (tid == 0) {
        for (uint32_t i = 0; i < 3; ++i) mbar_init(bar + 8 * i, 1);
        fence_mbar_init();
    }
    // position and cache rows are older than the predecessor (which wrote the queries): see pdl_wait
    const uint32_t pos = __ldcg(a.pos) + p.t0, seen = pos + p.rows / d.heads;
    uint32_t first, last;
    split_range(seen, split, p.splits, first, last);
    auto request = [&](uint32_t tile, uint32_t stage) {
        mbar_expect_tx(bar + 8 * stage, tile_bytes);
        for (uint32_t i = 0; i < panels; ++i)
            bulk_g2s(s_t + stage * tile_bytes + i * SP_N * 128, static_cast<const uint8_t *>(a.cache.p) + ((size_t)i * a.cache.ld + tile * SP_N) * 128, SP_N * 128, bar + 8 * stage);
    };
    auto landed = [&](uint32_t b, uint32_t parity) {
        bool ok = false;
        for (uint32_t spin = 0; spin < WAIT_LIMIT && !ok; ++spin) ok = mbar_try_wait(b, parity);
        if (!ok && a.err_flag != nullptr) atomicExch(a.err_flag, 1u);
    };
    if (tid == 0)
        for (uint32_t i = 0; i < p.stages && first + i < last; ++i) request(first + i, i);
    for (uint32_t i = tid; i < M; i += SP_THREADS) { s_m[i] = -INFINITY; s_l[i] = 0.0f; }
    pdl_wait();
    pdl_trigger();
    if (first < last) {
        if (tid == 0) {
            mbar_expect_tx(bar + 16, panels * M * 128);
            for (uint32_t i = 0; i < panels; ++i) bulk_g2s(s_q + i * M * 128, static_cast<const uint8_t *>(a.q_rows.p) + ((size_t)i * a.q_rows.ld + r0) * 128, M * 128, bar + 16);
        }
        __syncthreads();
        landed(bar + 16, 0);
    } else {
        __syncthreads();
    }
    float o[RB][U][2][4];
#pragma unroll
    for (int b = 0; b < RB; ++b)
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[b][u][0][e] = o[b][u][1][e] = 0.0f;
    const uint32_t units = d.rot_at / 16;
    const float scale = a.scale * LOG2E;
    for (uint32_t tile = first; tile < last; ++tile) {
        const uint32_t i = tile - first, stage = i % p.stages, st = s_t + stage * tile_bytes, j0 = tile * SP_N;
        landed(bar + 8 * stage, (i / p.stages) & 1u);
        float s[RB][4];
#pragma unroll
        for (int b = 0; b < RB; ++b) s[b][0] = s[b][1] = s[b][2] = s[b][3] = 0.0f;
        // panels are 64 columns: four 16-column steps, two per ldmatrix of the keys
        for (uint32_t k = 0; k < panels * 8; k += 4) {
            uint32_t b0, b1, b2, b3;
            ldsm4(tile_chunk(st, SP_N, warp * 8 + (lane & 7u), k + (lane >> 3)), b0, b1, b2, b3);
#pragma unroll
            for (int b = 0; b < RB; ++b) {
                uint32_t a0, a1, a2, a3;
                ldsm4(tile_chunk(s_q, M, b * 16 + (lane & 15u), k + (lane >> 4)), a0, a1, a2, a3);
                mma_bf16(s[b], a0, a1, a2, a3, b0, b1);
                ldsm4(tile_chunk(s_q, M, b * 16 + (lane & 15u), k + 2 + (lane >> 4)), a0, a1, a2, a3);
                mma_bf16(s[b], a0, a1, a2, a3, b2, b3);
            }
        }
#pragma unroll
        for (int b = 0; b < RB; ++b)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t row = b * 16 + (lane >> 2) + (e >> 1) * 8, j = warp * 8 + (lane & 3u) * 2 + (e & 1);
                const uint32_t qpos = pos + min(r0 + row, p.rows - 1) / d.heads;
                s_s[row * (SP_N + 4) + j] = j0 + j <= qpos ? s[b][e] * scale : -INFINITY;
            }
        __syncthreads();
#pragma unroll
        for (int q = 0; q < 2 * RB; ++q) {
            const uint32_t row = warp * 2 * RB + q;
            const float x = s_s[row * (SP_N + 4) + lane], y = s_s[row * (SP_N + 4) + 32 + lane];
            float mx = fmaxf(x, y);
#pragma unroll
            for (int k = 16; k > 0; k >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, k));
            const float m_old = s_m[row], m_new = fmaxf(m_old, mx), m_use = m_new == -INFINITY ? 0.0f : m_new;
            const float ex = exp2_approx(x - m_use), ey = exp2_approx(y - m_use), sum = warp_sum(ex + ey);
            g_p[row * (sp_pitch() / 2) + lane] = __float2bfloat16_rn(ex);
            g_p[row * (sp_pitch() / 2) + 32 + lane] = __float2bfloat16_rn(ey);
            if (lane == 0) {
                const float al = exp2_approx(m_old - m_use);
                s_al[row] = al;
                s_m[row] = m_new;
                s_l[row] = s_l[row] * al + sum;
            }
            __syncwarp();
        }
        __syncthreads();
#pragma unroll
        for (int b = 0; b < RB; ++b) {
            const float al0 = s_al[b * 16 + (lane >> 2)], al1 = s_al[b * 16 + 8 + (lane >> 2)];
#pragma unroll
            for (int u = 0; u < U; ++u)
#pragma unroll
                for (int n = 0; n < 2; ++n) { o[b][u][n][0] *= al0; o[b][u][n][1] *= al0; o[b][u][n][2] *= al1; o[b][u][n][3] *= al1; }
        }
#pragma unroll
        for (uint32_t k = 0; k < SP_N / 16; ++k) {
            uint32_t w[RB][4];
#pragma unroll
            for (int b = 0; b < RB; ++b) ldsm4(s_p + (b * 16 + (lane & 15u)) * sp_pitch() + k * 32 + (lane >> 4) * 16, w[b][0], w[b][1], w[b][2], w[b][3]);
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const uint32_t unit = warp + 8 * u;
                if (unit >= units) break;
                uint32_t b0, b1, b2, b3;
                ldsm4t(tile_chunk(st, SP_N, k * 16 + (lane & 15u), unit * 2 + (lane >> 4)), b0, b1, b2, b3);
#pragma unroll
                for (int b = 0; b < RB; ++b) {
                    mma_bf16(o[b][u][0], w[b][0], w[b][1], w[b][2], w[b][3], b0, b1);
                    mma_bf16(o[b][u][1], w[b][0], w[b][1], w[b][2], w[b][3], b2, b3);
                }
            }
        }
        __syncthreads();                     // everyone is done with the tile
        if (tid == 0 && tile + p.stages < last) request(tile + p.stages, stage);
    }
    for (uint32_t i = tid; i < n_row; i += SP_THREADS) {
        a.part_m[(size_t)(r0 + i) * p.splits + split] = s_m[i];
        a.part_l[(size_t)(r0 + i) * p.splits + split] = s_l[i];
    }
    if (first == last) return;               // the merge skips splits without a position
#pragma unroll
    for (int b = 0; b < RB; ++b)
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const uint32_t row = b * 16 + (lane >> 2) + ((e >> 1) & 1) * 8, k = (warp + 8 * u) * 16 + (e >> 2) * 8 + (lane & 3u) * 2 + (e & 1);
                if (row < n_row && k < d.kv_rank) a.part_o[((size_t)(r0 + row) * p.splits + split) * part_stride(d) + k] = o[b][u][e >> 2][e & 3];
            }
}

// fp32 (part_m in natural units, not log2): CTA = (split, row); scores by one warp per position, values by one thread per column
__global__ void __launch_bounds__(256) latent_split_f32_kernel(const SplitParams p) {
    extern __shared__ __align__(16) float sf[];
    const LatentAttnArgs &a = p.a;
    const LatentShape &d = a.d;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = blockIdx.y, split = blockIdx.x;
    float *s_q = sf, *s_o = s_q + d.row, *s_p = s_o + d.row;
    pdl_wait();
    pdl_trigger();
    const uint32_t pos = __ldcg(a.pos) + p.t0, seen = pos + row / d.heads + 1;
    uint32_t first, last;
    split_range(pos + p.rows / d.heads, split, p.splits, first, last);
    const float *q = static_cast<const float *>(a.q_rows.p) + (size_t)row * a.q_rows.ld, *cache = static_cast<const float *>(a.cache.p);
    for (uint32_t k = tid; k < d.row; k += 256) {
        s_q[k] = k < d.kv_rank || (k >= d.rot_at && k < d.rot_at + d.rot_dim) ? __ldcg(q + k) : 0.0f;
        s_o[k] = 0.0f;
    }
    float m = -INFINITY, l = 0.0f;
    __syncthreads();
    for (uint32_t tile = first; tile < last && tile * SP_N < seen; ++tile) {
        const uint32_t j0 = tile * SP_N, n = min(SP_N, seen - j0);
        for (uint32_t j = warp; j < n; j += 8) {
            const float *c = cache + (size_t)(j0 + j) * a.cache.ld;
            float s = 0.0f;
            for (uint32_t k = lane; k < d.row; k += 32) s = __fmaf_rn(s_q[k], __ldcg(c + k), s);
            s = warp_sum(s);
            if (lane == 0) s_p[j] = s * a.scale;
        }
        __syncthreads();
        float mx = -INFINITY;
        for (uint32_t j = 0; j < n; ++j) mx = fmaxf(mx, s_p[j]);
        const float m_new = fmaxf(m, mx), al = expf(m - m_new);
        __syncthreads();
        if (tid < n) s_p[tid] = expf(s_p[tid] - m_new);
        __syncthreads();
        float sum = 0.0f;
        for (uint32_t j = 0; j < n; ++j) sum += s_p[j];
        l = l * al + sum;
        m = m_new;
        for (uint32_t k = tid; k < d.kv_rank; k += 256) {
            float o = 0.0f;
            for (uint32_t j = 0; j < n; ++j) o = __fmaf_rn(s_p[j], __ldcg(cache + (size_t)(j0 + j) * a.cache.ld + k), o);
            s_o[k] = s_o[k] * al + o;
        }
        __syncthreads();
    }
    for (uint32_t k = tid; k < d.kv_rank; k += 256) a.part_o[((size_t)row * p.splits + split) * part_stride(d) + k] = s_o[k];
    if (tid == 0) { a.part_m[(size_t)row * p.splits + split] = m; a.part_l[(size_t)row * p.splits + split] = l; }
}

// grid (64 value rows, head, token): merge of the splits, then W_uv of the head.  Thread = (four columns, group of splits); the
// first partial results are requested before their factors are known, the weights before the dependency wait.
constexpr uint32_t VL_THREADS = 512, VL_PF = 8;
template <bool F32>
__global__ void __launch_bounds__(VL_THREADS) latent_value_kernel(const SplitParams p) {
    extern __shared__ __align__(16) float sf[];
    const LatentAttnArgs &a = p.a;
    const LatentShape &d = a.d;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, t = blockIdx.z, row = t * d.heads + h;
    const uint32_t panels = (d.kv_rank + PANEL - 1) / PANEL, padded = panels * PANEL, quads = part_stride(d) / 4;
    float *s_c = sf, *s_f = s_c + padded;
    float4 *s_part = reinterpret_cast<float4 *>(s_f + ((p.splits + 4) & ~3u));          // [VL_THREADS]
    for (uint32_t k = tid; k < padded; k += VL_THREADS) s_c[k] = 0.0f;
    const uint32_t sub = lane & 7u, v = blockIdx.x * 64 + warp * 4 + (lane >> 3), vv = min(v, d.vdim - 1);
    const uint32_t w_row = d.heads * latent_head_cols(d.dim) + h * latent_head_cols(d.vdim) + vv;
    const uint4 *wp = static_cast<const uint4 *>(a.kv_up.base) + (size_t)w_row * 8 + (sub ^ (w_row & 7u));
    uint4 w[VL_PF];
    if (!F32)
#pragma unroll
        for (uint32_t i = 0; i < VL_PF; ++i) w[i] = i < panels ? ldg_stream(wp + (size_t)i * a.kv_up.rows_pad * 8) : make_uint4(0, 0, 0, 0);
    pdl_wait();
    pdl_trigger();
    uint32_t first, last;                    // splits that hold a position at all
    const uint32_t seen = __ldcg(a.pos) + p.t0 + p.rows / d.heads;
    split_range(seen, 0, p.splits, first, last);
    const uint32_t used = min(p.splits, ((seen + SP_N - 1) / SP_N + last - 1) / max(1u, last));
    const float *pm = a.part_m + (size_t)row * p.splits, *pl = a.part_l + (size_t)row * p.splits;
    const float4 *po = reinterpret_cast<const float4 *>(a.part_o) + (size_t)row * p.splits * quads;
    // quads q0, q0 + cols, ..: `cols` threads side by side, `groups` of them over the splits
    const uint32_t cols = min(quads, VL_THREADS), groups = VL_THREADS / cols, g = tid / cols, q0 = tid % cols;
    constexpr uint32_t PRE = 4;
    float4 pre[PRE];
#pragma unroll
    for (uint32_t i = 0; i < PRE; ++i) pre[i] = g < groups && g + i * groups < used ? __ldcg(po + (size_t)(g + i * groups) * quads + q0) : make_float4(0, 0, 0, 0);
    if (warp == VL_THREADS / 32 - 1) {
        float m = -INFINITY, l = 0.0f;
        for (uint32_t s = lane; s < used; s += 32) m = fmaxf(m, __ldcg(pm + s));
#pragma unroll
        for (int k = 16; k > 0; k >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, k));
        for (uint32_t s = lane; s < used; s += 32) { const float f = F32 ? expf(__ldcg(pm + s) - m) : exp2f(__ldcg(pm + s) - m); s_f[s] = f; l = __fmaf_rn(f, __ldcg(pl + s), l); }
        l = warp_sum(l);
        if (lane == 0) s_f[p.splits] = 1.0f / l;
    }
    __syncthreads();
    const float inv = s_f[p.splits];
    for (uint32_t qb = 0; qb < quads; qb += cols) {
        const uint32_t q = qb + q0;
        float4 o = make_float4(0, 0, 0, 0);
        auto add = [&](float f, const float4 &x) { o.x = __fmaf_rn(f, x.x, o.x); o.y = __fmaf_rn(f, x.y, o.y); o.z = __fmaf_rn(f, x.z, o.z); o.w = __fmaf_rn(f, x.w, o.w); };
        if (g < groups && q < quads) {
            uint32_t s = g;
            if (qb == 0) {
#pragma unroll
                for (uint32_t i = 0; i < PRE; ++i, s += groups)
                    if (s < used) add(s_f[s], pre[i]);
            }
#pragma unroll 8
            for (; s < used; s += groups) add(s_f[s], __ldcg(po + (size_t)s * quads + q));
        }
        s_part[tid] = o;
        __syncthreads();
        if (tid < cols && q < quads) {
            for (uint32_t i = 1; i < groups; ++i) { const float4 x = s_part[i * cols + tid]; o.x += x.x; o.y += x.y; o.z += x.z; o.w += x.w; }
            const float e[4] = {o.x, o.y, o.z, o.w};
            for (uint32_t i = 0; i < 4 && q * 4 + i < d.kv_rank; ++i) s_c[q * 4 + i] = e[i] * inv;
        }
        __syncthreads();
    }
    float s = 0.0f;
    if (F32) {
        s = row_dot8<true>(a.kv_up, w_row, 0, panels, s_c, sub);
    } else {
#pragma unroll
        for (uint32_t i = 0; i < VL_PF; ++i)
            if (i < panels) s = dot8(w[i], s_c + i * PANEL + sub * 8, s);
        for (uint32_t i = VL_PF; i < panels; ++i) s = dot8(ldg_stream(wp + (size_t)i * a.kv_up.rows_pad * 8), s_c + i * PANEL + sub * 8, s);
#pragma unroll
        for (int m = 1; m < 8; m <<= 1) s = __fadd_rn(s, __shfl_xor_sync(0xffffffffu, s, m));
    }
    if (v < d.vdim && sub == 0) act_store<F32>(a.out, p.t0 + t, h * d.vdim + v, s);
}

// ------------------------------------------------------------------------------------------------ prompts, bf16
// queries as operand panels: per head the unrotated part, then the rotated one, each padded to whole panels with zeros; thread = one
// 16-byte chunk.  ALIGNED: rows and parts start at multiples of four floats.
template <bool ALIGNED>
__global__ void __launch_bounds__(256) latent_query_kernel(const LatentAttnArgs a, uint32_t n_tok) {
    const LatentShape &d = a.d;
    const uint32_t dc = latent_head_cols(d.dim), per = dc + latent_head_cols(d.rot_dim), t = blockIdx.y, chunks = d.heads * per / 8;
    pdl_wait();
    pdl_trigger();
    const float *cs = a.rot + (size_t)(__ldcg(a.pos) + t) * d.rot_dim;
    for (uint32_t i = blockIdx.x * 256 + threadIdx.x; i < chunks; i += gridDim.x * 256) {
        const uint32_t h = i / (per / 8), k = i % (per / 8) * 8;
        const bool rot = k >= dc;
        const uint32_t k0 = rot ? k - dc : k, n = rot ? d.rot_dim : d.dim;          // elements k0 .. k0 + 7 of a part of n
        const float *q = a.q + t * a.q_stride + h * (d.dim + d.rot_dim) + (rot ? d.dim : 0) + k0;
        float v[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
        if (ALIGNED && k0 + 8 <= n) {
            const float4 x = __ldcg(reinterpret_cast<const float4 *>(q)), y = __ldcg(reinterpret_cast<const float4 *>(q) + 1);
            v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
        } else {
#pragma unroll
            for (uint32_t j = 0; j < 8; ++j)
                if (k0 + j < n) v[j] = __ldcg(q + j);
        }
        if (rot)
#pragma unroll
            for (uint32_t j = 0; j < 8; j += 2)
                if (k0 + j < n) {
                    const float c = __ldg(cs + k0 + j), s = __ldg(cs + k0 + j + 1), x = v[j], y = v[j + 1];
                    v[j] = x * c - y * s;
                    v[j + 1] = y * c + x * s;
                }
        *reinterpret_cast<uint4 *>(static_cast<__nv_bfloat16 *>(a.q_rows.p) + panel_index(a.q_rows.ld, t, h * per + k)) =
            make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
    }
}

constexpr uint32_t FL_M = 128, FL_THREADS = 192, FL_HEADER = 1024;
struct FlashShape { uint32_t kt, pd, pr, pv, vn, tmem; size_t smem; };      // key tile, panels, padded value columns, tensor-memory columns
inline FlashShape flash_shape(const LatentShape &d) {
    FlashShape f{};
    f.pd = latent_head_cols(d.dim) / PANEL; f.pr = latent_head_cols(d.rot_dim) / PANEL; f.pv = latent_head_cols(d.vdim) / PANEL;
    f.vn = (d.vdim + 15u) & ~15u;
    for (uint32_t kt : {128u, 64u}) {
        f.kt = kt;
        f.smem = 1024 + FL_HEADER + (size_t)(f.pd + f.pr) * FL_M * 128 + (size_t)2 * (f.pd + f.pr + f.pv) * kt * 128;
        if (f.smem <= 226 * 1024) break;
    }
    f.tmem = 32;
    while (f.tmem < 2 * f.kt + f.vn) f.tmem *= 2;
    return f;
}

struct FlashParams {
    LatentAttnArgs a;
    uint32_t n_tok, pd, pr, pv, vn, tmem;
};

__device__ __forceinline__ uint64_t desc_k(uint32_t saddr) {       // K-major operand: eight-row groups 1024 bytes apart, 128-byte swizzle
    return (uint64_t)((saddr >> 4) & 0x3FFFu) | (1ull << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ uint64_t desc_mn(uint32_t saddr, uint32_t panel_bytes) {      // 64-column groups panel_bytes apart, eight-key groups 1024
    return (uint64_t)((saddr >> 4) & 0x3FFFu) | ((uint64_t)((panel_bytes >> 4) & 0x3FFFu) << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void mma_ss(uint32_t d_tmem, uint64_t desc_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t}\n"
        ::"r"(d_tmem), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(0u) : "memory");
}
__device__ __forceinline__ void mma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, {%5, %5, %5, %5}, p;\n\t}\n"
        ::"r"(d_tmem), "r"(a_tmem), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(0u) : "memory");
}
__device__ __forceinline__ void tc_commit(uint32_t bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
#define K2T_R8(v, i) "=r"(v[i]), "=r"(v[i + 1]), "=r"(v[i + 2]), "=r"(v[i + 3]), "=r"(v[i + 4]), "=r"(v[i + 5]), "=r"(v[i + 6]), "=r"(v[i + 7])
#define K2T_I8(v, i) "r"(v[i]), "r"(v[i + 1]), "r"(v[i + 2]), "r"(v[i + 3]), "r"(v[i + 4]), "r"(v[i + 5]), "r"(v[i + 6]), "r"(v[i + 7])
__device__ __forceinline__ void tm_ld32(uint32_t taddr, uint32_t *v) {      // 32 columns of the thread's lane; wait with tm_ld_wait
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
                 : K2T_R8(v, 0), K2T_R8(v, 8), K2T_R8(v, 16), K2T_R8(v, 24) : "r"(taddr) : "memory");
}
__device__ __forceinline__ void tm_st32(uint32_t taddr, const uint32_t *v) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x32.b32 [%32], {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31};"
                 ::K2T_I8(v, 0), K2T_I8(v, 8), K2T_I8(v, 16), K2T_I8(v, 24), "r"(taddr) : "memory");
}
__device__ __forceinline__ void tm_ld16(uint32_t taddr, uint32_t *v) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];" : K2T_R8(v, 0), K2T_R8(v, 8) : "r"(taddr) : "memory");
}
__device__ __forceinline__ void tm_st16(uint32_t taddr, const uint32_t *v) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%16], {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15};" ::K2T_I8(v, 0), K2T_I8(v, 8), "r"(taddr) : "memory");
}
__device__ __forceinline__ void tm_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tm_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void mbar_arrive(uint32_t bar) { asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory"); }
__device__ __forceinline__ bool fl_wait(uint32_t bar, uint32_t parity, volatile uint32_t *abort_w) {
    for (uint32_t spin = 0; spin < WAIT_LIMIT; ++spin) {
        if (mbar_try_wait(bar, parity)) return true;
        if ((spin & 255u) == 255u && *abort_w != 0) return false;
    }
    *abort_w = 1;
    return false;
}

// Warps 0 .. 3: softmax, one row (token) per thread; warp 4: bulk copies; warp 5: tensor-core issue.
// Tensor memory: S of even and odd tiles (KT columns each, the softmax weights overwrite them as bf16 pairs), then O.
template <int KT>
__global__ void __launch_bounds__(FL_THREADS, 1) latent_flash_kernel(const FlashParams p) {
    extern __shared__ uint8_t smem_raw[];
    const LatentAttnArgs &a = p.a;
    const LatentShape &d = a.d;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, t0 = (gridDim.x - 1 - blockIdx.x) * FL_M;      // longest rows first
    const uint32_t raw = (uint32_t)__cvta_generic_to_shared(smem_raw), sbase = (raw + 1023u) & ~1023u;
    uint8_t *smem = smem_raw + (sbase - raw);
    const uint32_t pq = p.pd + p.pr, k_bytes = pq * KT * 128, v_bytes = p.pv * KT * 128;
    const uint32_t s_q = sbase + FL_HEADER, s_k = s_q + pq * FL_M * 128, s_v = s_k + 2 * k_bytes;
    // barriers: queries, keys landed / free, values landed / free, S ready, weights ready, O updated, end
    const uint32_t b_q = sbase, b_kf = sbase + 8, b_ke = sbase + 24, b_vf = sbase + 40, b_ve = sbase + 56, b_s = sbase + 72, b_p = sbase + 88, b_o = sbase + 104, b_end = sbase + 112;
    volatile uint32_t *s_tmem = reinterpret_cast<volatile uint32_t *>(smem + 256), *s_abort = reinterpret_cast<volatile uint32_t *>(smem + 260);
    if (tid == 0) {
        mbar_init(b_q, 1);
        for (uint32_t i = 0; i < 2; ++i) {
            mbar_init(b_kf + 8 * i, 1); mbar_init(b_ke + 8 * i, 1); mbar_init(b_vf + 8 * i, 1); mbar_init(b_ve + 8 * i, 1);
            mbar_init(b_s + 8 * i, 1); mbar_init(b_p + 8 * i, 128);
        }
        mbar_init(b_o, 1);
        mbar_init(b_end, 1);
        *s_abort = 0;
        fence_mbar_init();
    }
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(sbase + 256), "r"(p.tmem) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *s_tmem, t_o = tmem + 2 * KT;
    pdl_wait();
    pdl_trigger();
    const uint32_t pos0 = __ldcg(a.pos), n_row = min(FL_M, p.n_tok - t0), n_tiles = (pos0 + t0 + n_row - 1) / KT + 1;

    if (warp == 4) {
        if (lane == 0) {
            const uint8_t *q = static_cast<const uint8_t *>(a.q_rows.p), *kv = static_cast<const uint8_t *>(a.kv.p), *cache = static_cast<const uint8_t *>(a.cache.p);
            mbar_expect_tx(b_q, pq * FL_M * 128);
            for (uint32_t i = 0; i < pq; ++i) bulk_g2s(s_q + i * FL_M * 128, q + ((size_t)(h * pq + i) * a.q_rows.ld + t0) * 128, FL_M * 128, b_q);
            auto keys = [&](uint32_t j) {
                const uint32_t b = j & 1u, dst = s_k + b * k_bytes;
                mbar_expect_tx(b_kf + 8 * b, k_bytes);
                for (uint32_t i = 0; i < p.pd; ++i) bulk_g2s(dst + i * KT * 128, kv + ((size_t)(h * p.pd + i) * a.kv.ld + j * KT) * 128, KT * 128, b_kf + 8 * b);
                for (uint32_t i = 0; i < p.pr; ++i) bulk_g2s(dst + (p.pd + i) * KT * 128, cache + ((size_t)(d.rot_at / PANEL + i) * a.cache.ld + j * KT) * 128, KT * 128, b_kf + 8 * b);
            };
            auto values = [&](uint32_t j) {
                const uint32_t b = j & 1u, dst = s_v + b * v_bytes;
                mbar_expect_tx(b_vf + 8 * b, v_bytes);
                for (uint32_t i = 0; i < p.pv; ++i) bulk_g2s(dst + i * KT * 128, kv + ((size_t)(d.heads * p.pd + h * p.pv + i) * a.kv.ld + j * KT) * 128, KT * 128, b_vf + 8 * b);
            };
            bool ok = true;
            uint32_t nk = 0, nv = 0;          // tiles requested
            for (uint32_t j = 0; j < n_tiles && ok; ++j) {
                if (j >= 2) ok = fl_wait(b_ke + 8 * (j & 1u), ((j >> 1) - 1u) & 1u, s_abort);
                if (!ok) break;
                keys(j);
                nk = j + 1;
                if (j >= 2) ok = fl_wait(b_ve + 8 * (j & 1u), ((j >> 1) - 1u) & 1u, s_abort);
                if (!ok) break;
                values(j);
                nv = j + 1;
            }
            if (!ok) {                        // copies in flight land before the CTA leaves
                if (a.err_flag != nullptr) atomicExch(a.err_flag, 1u);
                auto drain = [&](uint32_t bar, uint32_t parity) { for (uint32_t spin = 0; spin < WAIT_LIMIT && !mbar_try_wait(bar, parity); ++spin) {} };
                drain(b_q, 0);
                for (uint32_t j = nk > 2 ? nk - 2 : 0; j < nk; ++j) drain(b_kf + 8 * (j & 1u), (j >> 1) & 1u);
                for (uint32_t j = nv > 2 ? nv - 2 : 0; j < nv; ++j) drain(b_vf + 8 * (j & 1u), (j >> 1) & 1u);
            }
        }
    } else if (warp == 5) {
        if (lane == 0) {
            // fp32 accumulators, bf16 operands; A and B K-major for S, B with its columns consecutive for O
            const uint32_t id_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(KT >> 3) << 17) | ((FL_M >> 4) << 24);
            const uint32_t id_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((p.vn >> 3) << 17) | ((FL_M >> 4) << 24);
            const uint32_t steps_d = (d.dim + 15) / 16, steps_r = (d.rot_dim + 15) / 16;
            auto scores = [&](uint32_t j) {
                const uint32_t b = j & 1u, kb = s_k + b * k_bytes;
                if (!fl_wait(b_kf + 8 * b, (j >> 1) & 1u, s_abort)) return false;
                tc_fence_after();
                for (uint32_t i = 0; i < steps_d + steps_r; ++i) {
                    const uint32_t col = i < steps_d ? i * 16 : p.pd * PANEL + (i - steps_d) * 16, panel = col / PANEL, in = (col % PANEL) * 2;
                    mma_ss(tmem + b * KT, desc_k(s_q + panel * FL_M * 128 + in), desc_k(kb + panel * KT * 128 + in), id_s, i != 0 ? 1u : 0u);
                }
                tc_commit(b_s + 8 * b);
                tc_commit(b_ke + 8 * b);
                return true;
            };
            bool ok = fl_wait(b_q, 0, s_abort) && scores(0);
            for (uint32_t j = 0; j < n_tiles && ok; ++j) {
                const uint32_t b = j & 1u;
                if (j + 1 < n_tiles) {
                    if (j >= 1) ok = fl_wait(b_o, (j - 1) & 1u, s_abort);      // the weights of tile j - 1 lie where S of tile j + 1 goes
                    ok = ok && scores(j + 1);
                    if (!ok) break;
                }
                ok = fl_wait(b_p + 8 * b, (j >> 1) & 1u, s_abort) && fl_wait(b_vf + 8 * b, (j >> 1) & 1u, s_abort);
                if (!ok) break;
                tc_fence_after();
                for (uint32_t k = 0; k < KT / 16; ++k)
                    mma_ts(t_o, tmem + b * KT + k * 8, desc_mn(s_v + b * v_bytes + k * 16 * 128, KT * 128), id_o, (j | k) != 0 ? 1u : 0u);
                tc_commit(b_ve + 8 * b);
                tc_commit(b_o);
            }
            tc_commit(b_end);                 // also after a wait that gave up: completes when the issued products have
            if (!ok && a.err_flag != nullptr) atomicExch(a.err_flag, 1u);
            for (uint32_t spin = 0; spin < WAIT_LIMIT && !mbar_try_wait(b_end, 0u); ++spin) {}
        }
    } else {
        const uint32_t r = warp * 32 + lane, t = t0 + r, qpos = pos0 + min(t, p.n_tok - 1), lanes = (warp * 32u) << 16;
        const float sc = a.scale * LOG2E;
        float m = -INFINITY, l = 0.0f;         // maximum (of scores times sc) the weights are taken against, and their sum
        bool ok = true;
        for (uint32_t j = 0; j < n_tiles; ++j) {
            const uint32_t b = j & 1u, t_s = tmem + b * KT + lanes;
            ok = __all_sync(0xffffffffu, fl_wait(b_s + 8 * b, (j >> 1) & 1u, s_abort));
            if (!ok) break;
            tc_fence_after();
            uint32_t v[KT];
#pragma unroll
            for (int c = 0; c < KT; c += 32) tm_ld32(t_s + c, v + c);
            tm_ld_wait();
            if ((j + 1) * KT > pos0 + t0 + warp * 32) {          // some row of the warp does not see the whole tile
#pragma unroll
                for (int c = 0; c < KT; ++c)
                    if (j * KT + c > qpos) v[c] = 0xff800000u;
            }
            float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int c = 0; c < KT; ++c) mx[c & 3] = fmaxf(mx[c & 3], __uint_as_float(v[c]));
            const float m_new = fmaxf(m, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * sc);
            if (j == 0) {
                m = m_new;
            } else if (__any_sync(0xffffffffu, m_new > m + 8.0f)) {
                ok = __all_sync(0xffffffffu, fl_wait(b_o, (j - 1) & 1u, s_abort));
                if (!ok) break;
                tc_fence_after();
                const float al = exp2_approx(m - m_new);
                for (uint32_t c = 0; c < p.vn; c += 16) {
                    uint32_t o[16];
                    tm_ld16(t_o + lanes + c, o);
                    tm_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * al);
                    tm_st16(t_o + lanes + c, o);
                }
                l *= al;
                m = m_new;
            }
            float sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int c = 0; c < KT; c += 2) {
                const float x = exp2_approx(__fmaf_rn(__uint_as_float(v[c]), sc, -m)), y = exp2_approx(__fmaf_rn(__uint_as_float(v[c + 1]), sc, -m));
                sum[(c >> 1) & 3] += x + y;
                v[c >> 1] = pack_bf16(x, y);
            }
            l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
#pragma unroll
            for (int c = 0; c < KT / 2; c += 32) tm_st32(t_s + c, v + c);
            tm_st_wait();
            tc_fence_before();
            mbar_arrive(b_p + 8 * b);
        }
        // the last update by a barrier of its own: the phases of b_o may still be two behind here, and a parity tells only neighbours apart
        if (ok) ok = __all_sync(0xffffffffu, fl_wait(b_end, 0u, s_abort) && *s_abort == 0);
        tc_fence_after();
        if (ok) {
            const float inv = 1.0f / l;
            for (uint32_t c = 0; c < p.vn; c += 16) {
                uint32_t o[16];
                tm_ld16(t_o + lanes + c, o);
                tm_ld_wait();
                if (r < n_row) {
                    float f[16];
#pragma unroll
                    for (int i = 0; i < 16; ++i) f[i] = __uint_as_float(o[i]) * inv;
                    const uint32_t k = h * d.vdim + c;
                    if (c + 16 <= d.vdim && (k & 7u) == 0) {
#pragma unroll
                        for (int i = 0; i < 16; i += 8)
                            *reinterpret_cast<uint4 *>(static_cast<__nv_bfloat16 *>(a.out.p) + panel_index(a.out.ld, t, k + i)) =
                                make_uint4(pack_bf16(f[i], f[i + 1]), pack_bf16(f[i + 2], f[i + 3]), pack_bf16(f[i + 4], f[i + 5]), pack_bf16(f[i + 6], f[i + 7]));
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (c + i < d.vdim) act_store<false>(a.out, t, k + i, f[i]);
                    }
                }
            }
        } else if (lane == 0 && a.err_flag != nullptr) {
            atomicExch(a.err_flag, 1u);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 5) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(p.tmem) : "memory");
    }
}

// rows per CTA and stages of the split kernel: 0 when nothing fits
struct SplitShape { int rb; uint32_t stages; size_t smem; };
SplitShape split_shape(const LatentShape &d, uint32_t rows) {
    constexpr size_t MOST = 225 * 1024;
    if (d.rot_at > 1024) return SplitShape{0, 0, 0};
    if (rows > 16 && d.rot_at <= 512 && sp_smem<2>(d, 2) <= MOST) return SplitShape{2, 2, sp_smem<2>(d, 2)};
    for (uint32_t st : {2u, 1u})
        if (sp_smem<1>(d, st) <= MOST) return SplitShape{1, st, sp_smem<1>(d, st)};
    return SplitShape{0, 0, 0};
}

template <int RB, int U> cudaError_t split_launch_u(cudaStream_t s, const SplitParams &p, size_t smem, bool pdl) {
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(latent_split_kernel<RB, U>), smem);
    if (e != cudaSuccess) return e;
    return launch_kernel(latent_split_kernel<RB, U>, dim3(p.splits, (p.rows + 16 * RB - 1) / (16 * RB)), dim3(SP_THREADS), smem, s, pdl, p);
}
template <int RB> cudaError_t split_launch(cudaStream_t s, const SplitParams &p, size_t smem, bool pdl) {
    const uint32_t units = p.a.d.rot_at / 16;
    if (units <= 8) return split_launch_u<RB, 1>(s, p, smem, pdl);
    if (units <= 16) return split_launch_u<RB, 2>(s, p, smem, pdl);
    if (units <= 32) return split_launch_u<RB, 4>(s, p, smem, pdl);
    return RB == 1 ? split_launch_u<1, 8>(s, p, smem, pdl) : cudaErrorInvalidValue;
}

template <int KT> cudaError_t flash_launch(cudaStream_t s, const FlashParams &p, size_t smem, bool pdl) {
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(latent_flash_kernel<KT>), smem);
    if (e != cudaSuccess) return e;
    return launch_kernel(latent_flash_kernel<KT>, dim3((p.n_tok + FL_M - 1) / FL_M, p.a.d.heads), dim3(FL_THREADS), smem, s, pdl, p);
}

}  // namespace

LatentShape latent_shape(bool f32, uint32_t heads, uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t q_rank, uint32_t kv_rank) {
    LatentShape d{heads, dim, rot_dim, vdim, q_rank, kv_rank, 0, 0};
    d.rot_at = f32 ? (kv_rank + 3u) & ~3u : (kv_rank + 63u) & ~63u;
    d.row = d.rot_at + (f32 ? (rot_dim + 3u) & ~3u : (rot_dim + 63u) & ~63u);
    return d;
}

bool latent_attn_fits(bool f32, const LatentShape &d) {
    return f32 ? (size_t)(2 * d.row + SP_N) * 4 <= 200 * 1024 : split_shape(d, 1).rb != 0;
}
bool latent_flash_fits(const LatentShape &d) { const FlashShape f = flash_shape(d); return f.smem <= 226 * 1024 && f.vn <= 256 && f.tmem <= 512; }

cudaError_t launch_latent_prep(cudaStream_t s, bool f32, const LatentAttnArgs &a, uint32_t n_tok, bool pdl) {
    const uint32_t n = std::max(a.d.q_rank, a.d.kv_rank), threads = n_tok > 64 ? 256u : std::min(PREP_THREADS, std::max(64u, (n + 31u) & ~31u));
    return launch_kernel(f32 ? latent_prep_kernel<true> : latent_prep_kernel<false>, dim3(n_tok, 2), dim3(threads), 0, s, pdl, a);
}

uint32_t latent_splits(const LatentShape &d, uint32_t n_tok, uint32_t max_positions, int sm_count) {
    const uint32_t groups = (n_tok * d.heads + 31) / 32, tiles = (max_positions + SP_N - 1) / SP_N;
    return std::max(1u, std::min({(uint32_t)sm_count / std::max(1u, groups), tiles, 128u}));
}

cudaError_t launch_latent_few(cudaStream_t s, bool f32, const LatentAttnArgs &a, uint32_t t0, uint32_t n_tok, uint32_t splits, bool pdl) {
    const LatentShape &d = a.d;
    if (n_tok == 0 || n_tok > LATENT_TOKENS || splits == 0) return cudaErrorInvalidValue;
    SplitParams p{a, t0, n_tok * d.heads, splits, 0};
    const dim3 value_grid((d.vdim + 63) / 64, d.heads, n_tok);
    const size_t value_smem = ((size_t)((d.kv_rank + PANEL - 1) / PANEL) * PANEL + ((splits + 4) & ~3u) + 4 * VL_THREADS) * 4;
    cudaError_t e;
    if (f32) {
        e = launch_kernel(latent_absorb_f32_kernel, dim3((d.row + 255) / 256, d.heads, n_tok), dim3(256), 0, s, pdl, a, t0);
        if (e != cudaSuccess) return e;
        const size_t smem = (size_t)(2 * d.row + SP_N) * 4;
        e = allow_dynamic_smem(reinterpret_cast<const void *>(latent_split_f32_kernel), smem);
        if (e != cudaSuccess) return e;
        e = launch_kernel(latent_split_f32_kernel, dim3(splits, p.rows), dim3(256), smem, s, pdl, p);
        if (e != cudaSuccess) return e;
        return launch_kernel(latent_value_kernel<true>, value_grid, dim3(VL_THREADS), value_smem, s, pdl, p);
    }
    const uint32_t cols = d.rot_at / PANEL + 1;
    e = n_tok == 1 ? launch_kernel(latent_absorb_kernel<1>, dim3(cols, d.heads, 1), dim3(256), 0, s, pdl, a, t0, t0 + n_tok)
                   : launch_kernel(latent_absorb_kernel<4>, dim3(cols, d.heads, (n_tok + 3) / 4), dim3(256), 0, s, pdl, a, t0, t0 + n_tok);
    if (e != cudaSuccess) return e;
    const SplitShape sh = split_shape(d, p.rows);
    p.stages = sh.stages;
    e = sh.rb == 2 ? split_launch<2>(s, p, sh.smem, pdl) : sh.rb == 1 ? split_launch<1>(s, p, sh.smem, pdl) : cudaErrorInvalidValue;
    if (e != cudaSuccess) return e;
    return launch_kernel(latent_value_kernel<false>, value_grid, dim3(VL_THREADS), value_smem, s, pdl, p);
}

cudaError_t launch_latent_prompt(cudaStream_t s, const LatentAttnArgs &a, uint32_t n_tok, bool pdl) {
    const LatentShape &d = a.d;
    const FlashShape f = flash_shape(d);
    if (!latent_flash_fits(d) || n_tok > 65535u) return cudaErrorInvalidValue;
    const uint32_t chunks = d.heads * (latent_head_cols(d.dim) + latent_head_cols(d.rot_dim)) / 8;
    const bool aligned = d.dim % 4 == 0 && d.rot_dim % 4 == 0 && a.q_stride % 4 == 0;
    cudaError_t e = launch_kernel(aligned ? latent_query_kernel<true> : latent_query_kernel<false>, dim3(std::min(8u, (chunks + 255) / 256), n_tok), dim3(256), 0, s, pdl, a, n_tok);
    if (e != cudaSuccess) return e;
    const FlashParams p{a, n_tok, f.pd, f.pr, f.pv, f.vn, f.tmem};
    return f.kt == 128 ? flash_launch<128>(s, p, f.smem, pdl) : flash_launch<64>(s, p, f.smem, pdl);
}

}  // namespace k2t
