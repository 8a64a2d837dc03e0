// Products of dense matrices (k2t_dense.h for the storage): a bf16 GEMV for one to eight tokens per weight pass, a bf16 GEMM on
// the tensor cores (tcgen05.mma kind::f16, tensor-memory accumulators) for prompt batches, and fp32 forms of both on the CUDA
// cores for engines that run in true 32-bit.
#include <algorithm>
#include <cstdlib>

#include "k2t_dense.cuh"

namespace k2t {
namespace {

// ------------------------------------------------------------------------------------------------ bf16 GEMV
// A warp owns a group of eight rows and, with wk = 1 .. 8 warps per group, every wk-th panel of it: 1 KiB of consecutive
// weights per step.  Lane = (row pair r, r + 4; chunk c): both rows use the same eight activation values.  The first GV_PF
// panels are requested before the dependency wait, so a launch whose warps hold few panels has its whole matrix in flight
// while the predecessor still runs
// (four with four CTAs per SM, six with two: more bytes in flight where the rows give only few CTAs).
// ROWS: the output is fp32 rows.
template <int NT, int GV_PF, bool ROWS>
__global__ void __launch_bounds__(256, NT == 1 && GV_PF == 4 ? 4 : 2) dense_gemv_kernel(const uint4 *__restrict__ w, uint32_t rows, uint32_t rows_pad, uint32_t np, const uint4 *__restrict__ x,
                                                        uint32_t ld, uint32_t t0, uint32_t n_tok, const DenseOut out, uint32_t wk_log2) {
    __shared__ float s_part[8][8][NT];
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, wk = 1u << wk_log2, c = lane & 7u, r = lane >> 3;
    const uint32_t group = blockIdx.x * (8u >> wk_log2) + (warp >> wk_log2), ks = warp & (wk - 1);
    const bool live = group * 8 < rows;
    const size_t pitch = (size_t)rows_pad * 8;
    const uint4 *w0 = w + (size_t)group * 64 + r * 8 + (c ^ r), *w1 = w + (size_t)group * 64 + (r + 4) * 8 + (c ^ (r + 4));
    uint4 a[GV_PF], b[GV_PF];
#pragma unroll
    for (uint32_t i = 0; i < GV_PF; ++i) {
        const uint32_t p = ks + i * wk;
        if (live && p < np) { a[i] = ldg_stream(w0 + p * pitch); b[i] = ldg_stream(w1 + p * pitch); }
    }
    pdl_wait();
    pdl_trigger();
    float acc0[NT], acc1[NT];
#pragma unroll
    for (int t = 0; t < NT; ++t) acc0[t] = acc1[t] = 0.0f;
    if (live)
        for (uint32_t p0 = ks; p0 < np; p0 += GV_PF * wk)
#pragma unroll
            for (uint32_t i = 0; i < GV_PF; ++i) {
                const uint32_t p = p0 + i * wk;
                if (p >= np) break;
                const uint4 u = a[i], v = b[i];
                const uint32_t pn = p + GV_PF * wk;
                if (pn < np) { a[i] = ldg_stream(w0 + pn * pitch); b[i] = ldg_stream(w1 + pn * pitch); }
#pragma unroll
                for (int t = 0; t < NT; ++t) {
                    const uint4 q = x[((size_t)p * ld + t0 + t) * 8 + (c ^ ((t0 + t) & 7u))];
                    const float x0 = bf_lo(q.x), x1 = bf_hi(q.x), x2 = bf_lo(q.y), x3 = bf_hi(q.y), x4 = bf_lo(q.z), x5 = bf_hi(q.z), x6 = bf_lo(q.w), x7 = bf_hi(q.w);
                    float s = acc0[t];
                    s = __fmaf_rn(bf_lo(u.x), x0, s); s = __fmaf_rn(bf_hi(u.x), x1, s); s = __fmaf_rn(bf_lo(u.y), x2, s); s = __fmaf_rn(bf_hi(u.y), x3, s);
                    s = __fmaf_rn(bf_lo(u.z), x4, s); s = __fmaf_rn(bf_hi(u.z), x5, s); s = __fmaf_rn(bf_lo(u.w), x6, s); s = __fmaf_rn(bf_hi(u.w), x7, s);
                    acc0[t] = s;
                    s = acc1[t];
                    s = __fmaf_rn(bf_lo(v.x), x0, s); s = __fmaf_rn(bf_hi(v.x), x1, s); s = __fmaf_rn(bf_lo(v.y), x2, s); s = __fmaf_rn(bf_hi(v.y), x3, s);
                    s = __fmaf_rn(bf_lo(v.z), x4, s); s = __fmaf_rn(bf_hi(v.z), x5, s); s = __fmaf_rn(bf_lo(v.w), x6, s); s = __fmaf_rn(bf_hi(v.w), x7, s);
                    acc1[t] = s;
                }
            }
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int m = 1; m < 8; m <<= 1) {
            acc0[t] = __fadd_rn(acc0[t], __shfl_xor_sync(0xffffffffu, acc0[t], m));
            acc1[t] = __fadd_rn(acc1[t], __shfl_xor_sync(0xffffffffu, acc1[t], m));
        }
    if (c == 0)
#pragma unroll
        for (int t = 0; t < NT; ++t) { s_part[warp][r][t] = acc0[t]; s_part[warp][r + 4][t] = acc1[t]; }
    __syncthreads();
    // thread = (group of the CTA, row, token)
    const uint32_t groups = 8u >> wk_log2;
    for (uint32_t i = threadIdx.x; i < groups * 8 * NT; i += 256) {
        const uint32_t row_l = i & 7u, g = (i >> 3) % groups, t = (i >> 3) / groups;
        const uint32_t row = (blockIdx.x * groups + g) * 8 + row_l;
        if (row >= rows || t0 + t >= n_tok) continue;
        float s = 0.0f, s1 = 0.0f;
        for (uint32_t k = 0; k < wk; ++k) s = __fadd_rn(s, s_part[g * wk + k][row_l][t]);
        if (ROWS) {
            out.rows[(size_t)(t0 + t) * out.stride + row] = s;
            continue;
        }
        if (out.kind == Epi::GeluGated && (row_l & 1u) == 0)
            for (uint32_t k = 0; k < wk; ++k) s1 = __fadd_rn(s1, s_part[g * wk + k][row_l + 1][t]);
        dense_store<false>(out, t0 + t, row, s, s1);
    }
}

template <int NT>
cudaError_t gemv_nt(cudaStream_t s, const DenseView &m, const Act &x, uint32_t t0, uint32_t n_tok, const DenseOut &out, int sm_count, bool pdl) {
    const uint32_t groups = (m.rows + 7) / 8;
    // warps per row group: the fewest rounds of panels over the waves of the grid (a CTA beyond a full wave costs a whole round)
    const uint32_t slots = (uint32_t)sm_count * (NT == 1 ? 4u : 2u);
    uint32_t wl = 0;
    float best = 1e30f;
    for (uint32_t l = 0; l <= 3 && (1u << l) <= m.panels; ++l) {
        const uint32_t ctas = (groups + (8u >> l) - 1) / (8u >> l), waves = (ctas + slots - 1) / slots, steps = (m.panels + (1u << l) - 1) >> l;
        // a step's time grows with the warps that share an SM's bandwidth, and has a floor of its own
        const float fill = (float)ctas / (float)(waves * slots), t = (float)waves * (3.0f + (float)steps * (0.35f + 0.65f * fill));
        if (t < best) { best = t; wl = l; }
    }
    const uint32_t per = 8u >> wl, ctas = (groups + per - 1) / per;
    const bool deep = NT == 1 && ctas <= 2u * (uint32_t)sm_count;
    constexpr int DEEP = NT == 1 ? 6 : 4;
    auto k = out.kind == Epi::Rows ? (deep ? dense_gemv_kernel<NT, DEEP, true> : dense_gemv_kernel<NT, 4, true>) : deep ? dense_gemv_kernel<NT, DEEP, false> : dense_gemv_kernel<NT, 4, false>;
    return launch_kernel(k, dim3(ctas), dim3(256), 0, s, pdl, static_cast<const uint4 *>(m.base), m.rows, m.rows_pad, m.panels,
                         static_cast<const uint4 *>(x.p), x.ld, t0, n_tok, out, wl);
}

// ------------------------------------------------------------------------------------------------ bf16 GEMM (tensor cores)
// CTA = 128 rows x NT tokens.  Warp 4 streams operand tiles (one bulk copy of 16 KiB of weights and one of NT x 128 bytes of
// activations per 64 columns; both lie in the operand layout already, so nothing touches them on the way), warp 5 issues four
// tcgen05.mma (K 16 each) per stage and commits the stage back, warps 0 .. 3 and 6 .. 9 read the accumulators out of tensor memory
// (lane = row, a quarter of the rows per warp, every second stretch of 32 tokens) and store: 32 consecutive outputs of a token per
// warp store.
constexpr uint32_t GM_THREADS = 320;
constexpr uint32_t GM_A = DENSE_ROW_TILE * PANEL * 2;
constexpr uint32_t GM_HEADER = 1024;
constexpr uint32_t GM_WAIT_LIMIT = 1u << 22;
template <int NT> __host__ __device__ constexpr uint32_t gm_stages() { return NT == 256 ? 4u : NT == 128 ? 3u : 4u; }
template <int NT> __host__ __device__ constexpr uint32_t gm_smem() { return GM_HEADER + 1024 + gm_stages<NT>() * (GM_A + NT * PANEL * 2); }

struct GemmArgs {
    const uint8_t *w, *x;
    uint32_t rows, rows_pad, np, ld, n_tok;
    DenseOut out;
    uint32_t *err_flag;
    const void *const *bases;           // GROUPED: images of the experts, blockIdx.y = item
    const ExpertItem *items;
    const uint32_t *n_items;
};

__device__ __forceinline__ bool gm_wait(uint32_t bar, uint32_t parity, volatile uint32_t *abort_w) {
    for (uint32_t spin = 0; spin < GM_WAIT_LIMIT; ++spin) {
        if (mbar_try_wait(bar, parity)) return true;
        if ((spin & 255u) == 255u && *abort_w != 0) return false;
    }
    *abort_w = 1;
    return false;
}
__device__ __forceinline__ uint64_t gm_desc(uint32_t saddr) {
    // start address, (unused) leading offset 1, stride of eight rows 1024 bytes, descriptor version 1, 128-byte swizzle
    return (uint64_t)((saddr >> 4) & 0x3FFFu) | (1ull << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void gm_mma(uint32_t d_tmem, uint64_t desc_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t"
        ".reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t"
        "}\n" ::"r"(d_tmem), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(0u) : "memory");
}
__device__ __forceinline__ void gm_commit(uint32_t bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void gm_ld32(uint32_t taddr, uint32_t (&v)[32]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];\n\t"
        "tcgen05.wait::ld.sync.aligned;"
        : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]),
          "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]), "=r"(v[16]), "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]),
          "=r"(v[24]), "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
        : "r"(taddr) : "memory");
}

// 32 sums per lane (lane = row, registers = tokens tok .. tok + n - 1, tok a multiple of eight) -> output.  Activations: neighbouring
// lanes swap halves, so that a lane stores two columns (or one product of a pair) of every second token.  FULL: no token and no
// row of the warp is beyond the end - stores without predicates, which take a fraction of the instructions.
template <bool FULL> __device__ __forceinline__ void gm_store_part(const DenseOut &o, uint32_t rows, uint32_t row, uint32_t tok, uint32_t n, uint32_t (&v)[32]) {
    if (o.kind == Epi::Rows || o.kind == Epi::Softcap) {
        if (!FULL && row >= rows) return;
        float *p = o.rows + (size_t)tok * o.stride + row;
        const uint32_t stride = (uint32_t)o.stride;
        if (o.kind == Epi::Rows) {
#pragma unroll
            for (uint32_t t = 0; t < 32; ++t)
                if (FULL || t < n) p[t * stride] = __uint_as_float(v[t]);
        } else {
#pragma unroll
            for (uint32_t t = 0; t < 32; ++t)
                if (FULL || t < n) p[t * stride] = softcap(__uint_as_float(v[t]), o.cap);
        }
        return;
    }
    const uint32_t odd = threadIdx.x & 1u, r = row & ~1u, k = o.kind == Epi::GeluGated ? r >> 1 : r, chunk = ((k >> 3) & 7u) ^ odd;
    // element of (token tok + odd + t, column k) for even t: its chunk is chunk ^ (t & 7)
    __nv_bfloat16 *p = static_cast<__nv_bfloat16 *>(o.act.p) + ((size_t)(k >> 6) * o.act.ld + tok + odd) * PANEL + (k & 7u);
#pragma unroll
    for (uint32_t t = 0; t < 32; t += 2) {
        const float mine = __uint_as_float(odd ? v[t + 1] : v[t]), other = __shfl_xor_sync(0xffffffffu, __uint_as_float(odd ? v[t] : v[t + 1]), 1);
        const float lo = odd ? other : mine, hi = odd ? mine : other;       // rows r and r + 1 of the token
        if (!FULL && (t + odd >= n || r >= rows)) continue;
        __nv_bfloat16 *q = p + t * PANEL + ((chunk ^ (t & 7u)) << 3);
        if (o.kind == Epi::GeluGated) {
            *q = __float2bfloat16_rn(gelu_tanh_fast(lo) * hi);
        } else {
            const float x = o.kind == Epi::Relu2 ? relu_squared(lo) : lo, y = o.kind == Epi::Relu2 ? relu_squared(hi) : hi;
            if (FULL || r + 1 < rows) *reinterpret_cast<uint32_t *>(q) = pack_bf16(x, y);
            else *q = __float2bfloat16_rn(x);
        }
    }
}
__device__ __forceinline__ void gm_store(const DenseOut &o, uint32_t rows, uint32_t row, uint32_t tok, uint32_t n, uint32_t (&v)[32]) {
    if (n == 32 && (row | 31u) < rows) gm_store_part<true>(o, rows, row, tok, n, v);
    else gm_store_part<false>(o, rows, row, tok, n, v);
}

template <int NT, bool GROUPED>
__global__ void __launch_bounds__(GM_THREADS) dense_gemm_kernel(const GemmArgs a) {
    extern __shared__ uint8_t smem_raw[];
    constexpr uint32_t S = gm_stages<NT>(), B_BYTES = NT * PANEL * 2;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t row0 = blockIdx.x * DENSE_ROW_TILE;
    uint32_t tok0 = blockIdx.y * NT, tok_end = a.n_tok;
    const uint8_t *w = a.w;
    if (GROUPED) {                       // the items come from the predecessor
        pdl_wait();
        if (blockIdx.y >= __ldcg(a.n_items)) return;
        const ExpertItem it = a.items[blockIdx.y];
        tok0 = it.row0;
        tok_end = it.row_end;
        w = static_cast<const uint8_t *>(a.bases[it.expert]);
    }
    const uint32_t raw = (uint32_t)__cvta_generic_to_shared(smem_raw), sbase = (raw + 1023u) & ~1023u;
    uint8_t *smem = smem_raw + (sbase - raw);
    const uint32_t bar_full = sbase, bar_empty = sbase + 64, bar_done = sbase + 128;
    volatile uint32_t *s_tmem = reinterpret_cast<volatile uint32_t *>(smem + 256);
    volatile uint32_t *s_abort = reinterpret_cast<volatile uint32_t *>(smem + 260);
    const uint32_t a_base = sbase + GM_HEADER, b_base = a_base + S * GM_A;
    if (tid == 0) {
        for (uint32_t i = 0; i < S; ++i) { mbar_init(bar_full + 8 * i, 1); mbar_init(bar_empty + 8 * i, 1); }
        mbar_init(bar_done, 1);
        *s_abort = 0;
        fence_mbar_init();
    }
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(sbase + 256), "r"((uint32_t)NT) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *s_tmem;

    if (warp == 4) {
        if (lane == 0) {
            const uint8_t *wsrc = w + (size_t)row0 * (PANEL * 2), *xsrc = a.x + (size_t)tok0 * (PANEL * 2);
            const size_t w_pitch = (size_t)a.rows_pad * (PANEL * 2), x_pitch = (size_t)a.ld * (PANEL * 2);
            const uint32_t pre = min(S, a.np);
            for (uint32_t p = 0; p < pre; ++p) {            // the weights do not depend on the predecessor
                mbar_expect_tx(bar_full + 8 * p, GM_A + B_BYTES);
                bulk_g2s(a_base + p * GM_A, wsrc + p * w_pitch, GM_A, bar_full + 8 * p);
            }
            pdl_wait();
            pdl_trigger();
            for (uint32_t p = 0; p < pre; ++p) bulk_g2s(b_base + p * B_BYTES, xsrc + p * x_pitch, B_BYTES, bar_full + 8 * p);
            bool ok = true;
            uint32_t issued = pre;
            for (uint32_t p = pre; p < a.np && ok; ++p) {
                const uint32_t s = p % S;
                ok = gm_wait(bar_empty + 8 * s, ((p / S) - 1u) & 1u, s_abort);
                if (!ok) break;
                mbar_expect_tx(bar_full + 8 * s, GM_A + B_BYTES);
                bulk_g2s(a_base + s * GM_A, wsrc + p * w_pitch, GM_A, bar_full + 8 * s);
                bulk_g2s(b_base + s * B_BYTES, xsrc + p * x_pitch, B_BYTES, bar_full + 8 * s);
                issued = p + 1;
            }
            if (!ok) {
                if (a.err_flag != nullptr) atomicExch(a.err_flag, 1u);
                for (uint32_t p = issued > S ? issued - S : 0; p < issued; ++p)        // copies in flight land before the CTA leaves
                    for (uint32_t spin = 0; spin < GM_WAIT_LIMIT && !mbar_try_wait(bar_full + 8 * (p % S), (p / S) & 1u); ++spin) {}
            }
        }
    } else if (warp == 5) {
        if (lane == 0) {
            // fp32 accumulators, bf16 A and B, both K-major, N / 8, M / 16
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NT >> 3) << 17) | ((DENSE_ROW_TILE >> 4) << 24);
            bool ok = true;
            for (uint32_t p = 0; p < a.np; ++p) {
                const uint32_t s = p % S;
                ok = gm_wait(bar_full + 8 * s, (p / S) & 1u, s_abort);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint64_t da = gm_desc(a_base + s * GM_A), db = gm_desc(b_base + s * B_BYTES);
#pragma unroll
                for (uint32_t k = 0; k < 4; ++k) gm_mma(tmem, da + 2 * k, db + 2 * k, idesc, (p | k) != 0 ? 1u : 0u);
                gm_commit(bar_empty + 8 * s);
            }
            gm_commit(bar_done);          // also after a wait that gave up: completes when the issued products have
            if (!ok && a.err_flag != nullptr) atomicExch(a.err_flag, 1u);
        }
    } else {
        pdl_wait();
        bool ok = false;
        for (uint32_t spin = 0; spin < 8 * GM_WAIT_LIMIT && !ok; ++spin) ok = mbar_try_wait(bar_done, 0u);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        ok = ok && *s_abort == 0;
        if (!ok && lane == 0 && a.err_flag != nullptr) atomicExch(a.err_flag, 1u);
        const uint32_t quarter = warp & 3u, row = row0 + quarter * 32 + lane;          // a warp reaches the tensor-memory lanes of its number mod 4
#pragma unroll 1
        for (uint32_t c = warp < 4 ? 0 : 32; c < NT; c += 64) {
            if (tok0 + c >= tok_end || !ok) break;
            uint32_t v[32];
            gm_ld32(tmem + ((quarter * 32u) << 16) + c, v);
            gm_store(a.out, a.rows, row, tok0 + c, min(32u, tok_end - tok0 - c), v);
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 5) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((uint32_t)NT) : "memory");
    }
}

template <int NT> cudaError_t gemm_nt(cudaStream_t s, const GemmArgs &a, bool pdl) {
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(dense_gemm_kernel<NT, false>), gm_smem<NT>());
    if (e != cudaSuccess) return e;
    return launch_kernel(dense_gemm_kernel<NT, false>, dim3(a.rows_pad / DENSE_ROW_TILE, (a.n_tok + NT - 1) / NT), dim3(GM_THREADS), gm_smem<NT>(), s, pdl, a);
}

// ------------------------------------------------------------------------------------------------ fp32
template <int NT>
__global__ void __launch_bounds__(256) dense_gemv_f32_kernel(const float *__restrict__ w, uint32_t rows, uint32_t ldw, const float *__restrict__ x, uint32_t ldx,
                                                            uint32_t n_tok, float *__restrict__ out, size_t out_stride) {
    const uint32_t lane = threadIdx.x & 31, row = blockIdx.x * 8 + (threadIdx.x >> 5), t0 = blockIdx.y * NT;
    pdl_wait();
    pdl_trigger();
    if (row >= rows) return;
    float acc[NT];
#pragma unroll
    for (int t = 0; t < NT; ++t) acc[t] = 0.0f;
    for (uint32_t k = lane * 4; k < ldw; k += 128) {
        const float4 u = __ldg(reinterpret_cast<const float4 *>(w + (size_t)row * ldw + k));
#pragma unroll
        for (int t = 0; t < NT; ++t) {
            if (t0 + t >= n_tok) break;
            const float4 v = *reinterpret_cast<const float4 *>(x + (size_t)(t0 + t) * ldx + k);
            acc[t] = __fmaf_rn(u.x, v.x, acc[t]); acc[t] = __fmaf_rn(u.y, v.y, acc[t]); acc[t] = __fmaf_rn(u.z, v.z, acc[t]); acc[t] = __fmaf_rn(u.w, v.w, acc[t]);
        }
    }
#pragma unroll
    for (int t = 0; t < NT; ++t) {
        const float s = warp_sum(acc[t]);
        if (lane == 0 && t0 + t < n_tok) out[(size_t)(t0 + t) * out_stride + row] = s;
    }
}

// 64 rows x 64 tokens per CTA, 16 columns per step, 4 x 4 outputs per thread
__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const float *__restrict__ w, uint32_t rows, uint32_t ldw, const float *__restrict__ x, uint32_t ldx,
                                                            uint32_t n_tok, float *__restrict__ out, size_t out_stride) {
    __shared__ float s_w[16][68], s_x[16][68];
    const uint32_t tid = threadIdx.x, row0 = blockIdx.x * 64, tok0 = blockIdx.y * 64, li = tid >> 2, lk = (tid & 3u) * 4, tr = tid & 15u, tt = tid >> 4;
    pdl_wait();
    pdl_trigger();
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < ldw; k0 += 16) {
        float4 u = make_float4(0, 0, 0, 0), v = u;
        if (k0 + lk < ldw) {
            if (row0 + li < rows) u = __ldg(reinterpret_cast<const float4 *>(w + (size_t)(row0 + li) * ldw + k0 + lk));
            if (tok0 + li < n_tok) v = *reinterpret_cast<const float4 *>(x + (size_t)(tok0 + li) * ldx + k0 + lk);
        }
        __syncthreads();
        s_w[lk][li] = u.x; s_w[lk + 1][li] = u.y; s_w[lk + 2][li] = u.z; s_w[lk + 3][li] = u.w;
        s_x[lk][li] = v.x; s_x[lk + 1][li] = v.y; s_x[lk + 2][li] = v.z; s_x[lk + 3][li] = v.w;
        __syncthreads();
#pragma unroll
        for (uint32_t k = 0; k < 16; ++k) {
            float a[4], b[4];
#pragma unroll
            for (uint32_t i = 0; i < 4; ++i) { a[i] = s_w[k][tr + 16 * i]; b[i] = s_x[k][tt * 4 + i]; }
#pragma unroll
            for (uint32_t i = 0; i < 4; ++i)
#pragma unroll
                for (uint32_t j = 0; j < 4; ++j) acc[i][j] = __fmaf_rn(a[i], b[j], acc[i][j]);
        }
    }
#pragma unroll
    for (uint32_t j = 0; j < 4; ++j) {
        const uint32_t t = tok0 + tt * 4 + j;
        if (t >= n_tok) break;
#pragma unroll
        for (uint32_t i = 0; i < 4; ++i)
            if (row0 + tr + 16 * i < rows) out[(size_t)t * out_stride + row0 + tr + 16 * i] = acc[i][j];
    }
}

__global__ void __launch_bounds__(256) dense_epilogue_f32_kernel(uint32_t rows, uint32_t n_tok, const DenseOut out) {
    pdl_wait();
    pdl_trigger();
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < (size_t)n_tok * rows; i += (size_t)gridDim.x * 256) {
        const uint32_t t = (uint32_t)(i / rows), r = (uint32_t)(i % rows);
        const float *p = out.rows + (size_t)t * out.stride + r;
        dense_store<true>(out, t, r, *p, out.kind == Epi::GeluGated && r + 1 < rows ? p[1] : 0.0f);
    }
}

template <bool F32>
__global__ void __launch_bounds__(256) dense_pack_kernel(const float *__restrict__ x, uint32_t n_tok, uint32_t cols, uint32_t padded, const Act out) {
    pdl_wait();
    pdl_trigger();
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < (size_t)n_tok * padded; i += (size_t)gridDim.x * 256) {
        const uint32_t t = (uint32_t)(i / padded), k = (uint32_t)(i % padded);
        act_store<F32>(out, t, k, k < cols ? x[(size_t)t * cols + k] : 0.0f);
    }
}

}  // namespace

cudaError_t launch_dense_pack(cudaStream_t s, bool f32, const float *x, uint32_t n_tok, uint32_t cols, const Act &out, bool pdl) {
    const uint32_t padded = f32 ? dense_f32_ld(cols) : dense_panels(cols) * PANEL;
    const uint32_t ctas = (uint32_t)std::min<size_t>(1184, ((size_t)n_tok * padded + 255) / 256);
    return launch_kernel(f32 ? dense_pack_kernel<true> : dense_pack_kernel<false>, dim3(ctas), dim3(256), 0, s, pdl, x, n_tok, cols, padded, out);
}

cudaError_t launch_dense_out(cudaStream_t s, const DeviceMatrix &dm, const Act &x, uint32_t n_tok, const DenseOut &out, int sm_count, uint32_t *err_flag,
                             uint32_t *launches, bool pdl) {
    const DenseView m = dense_view(dm);
    *launches = 0;
    if (n_tok == 0) return cudaSuccess;
    if (dm.geom.fmt == FMT_DENSE32) {
        *launches = out.kind == Epi::Rows ? 1 : 2;
        const float *w = static_cast<const float *>(m.base), *xv = static_cast<const float *>(x.p);
        const cudaError_t e = n_tok < 16 ? launch_kernel(dense_gemv_f32_kernel<4>, dim3((m.rows + 7) / 8, (n_tok + 3) / 4), dim3(256), 0, s, pdl, w, m.rows, m.rows_pad, xv, x.ld, n_tok, out.rows, out.stride)
                                         : launch_kernel(dense_gemm_f32_kernel, dim3((m.rows + 63) / 64, (n_tok + 63) / 64), dim3(256), 0, s, pdl, w, m.rows, m.rows_pad, xv, x.ld, n_tok, out.rows, out.stride);
        if (e != cudaSuccess || out.kind == Epi::Rows) return e;
        return launch_kernel(dense_epilogue_f32_kernel, dim3((uint32_t)std::min<size_t>(1184, ((size_t)n_tok * m.rows + 255) / 256)), dim3(256), 0, s, pdl, m.rows, n_tok, out);
    }
    if (dm.geom.fmt != FMT_DENSE16) return cudaErrorInvalidValue;
    if (n_tok >= DENSE_TC_MIN) {
        const GemmArgs a{static_cast<const uint8_t *>(m.base), static_cast<const uint8_t *>(x.p), m.rows, m.rows_pad, m.panels, x.ld, n_tok, out, err_flag, nullptr, nullptr, nullptr};
        // token tile by the time of the grid's waves (measured, in units of a 256-token wave): tiles up to 128 tokens run two CTAs
        // per SM, so that one's stores overlap the other's products; activations cost the store phase more than fp32 rows
        static const struct { uint32_t nt; float alone, wave; } tiles[4] = {{256, 1.0f, 1.0f}, {128, 0.88f, 1.12f}, {64, 0.86f, 0.78f}, {32, 0.85f, 0.70f}};
        uint32_t best = 32;
        float best_t = 1e30f;
        for (const auto &c : tiles) {
            const uint32_t ctas = (m.rows_pad / DENSE_ROW_TILE) * ((n_tok + c.nt - 1) / c.nt), slots = (uint32_t)sm_count * (c.nt == 256 ? 1u : 2u);
            float t = ctas <= (uint32_t)sm_count ? c.alone : (float)((ctas + slots - 1) / slots) * c.wave;
            if (c.nt == 256 && out.kind != Epi::Rows) t *= 1.15f;
            if (t < best_t) { best_t = t; best = c.nt; }
        }
        *launches = 1;
        return best == 256 ? gemm_nt<256>(s, a, pdl) : best == 128 ? gemm_nt<128>(s, a, pdl) : best == 64 ? gemm_nt<64>(s, a, pdl) : gemm_nt<32>(s, a, pdl);
    }
    // weight passes of up to eight tokens (rows of the activation are padded to eight: a pass may read, never store, beyond n_tok)
    for (uint32_t t0 = 0; t0 < n_tok; t0 += 8) {
        const uint32_t left = n_tok - t0;
        const cudaError_t e = left > 4 ? gemv_nt<8>(s, m, x, t0, n_tok, out, sm_count, pdl) : left > 2 ? gemv_nt<4>(s, m, x, t0, n_tok, out, sm_count, pdl)
                              : left == 2 ? gemv_nt<2>(s, m, x, t0, n_tok, out, sm_count, pdl) : gemv_nt<1>(s, m, x, t0, n_tok, out, sm_count, pdl);
        *launches += 1;
        if (e != cudaSuccess) return e;
    }
    return cudaSuccess;
}

template <int NT> static cudaError_t gemm_experts_nt(cudaStream_t s, const GemmArgs &a, uint32_t max_items, bool pdl) {
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(dense_gemm_kernel<NT, true>), gm_smem<NT>());
    if (e != cudaSuccess) return e;
    return launch_kernel(dense_gemm_kernel<NT, true>, dim3(a.rows_pad / DENSE_ROW_TILE, max_items), dim3(GM_THREADS), gm_smem<NT>(), s, pdl, a);
}
cudaError_t launch_dense_experts(cudaStream_t s, const ExpertView &m, const Act &x, const ExpertItem *items, const uint32_t *n_items, uint32_t max_items,
                                 uint32_t tile, const DenseOut &out, uint32_t *err_flag, bool pdl) {
    if (max_items == 0 || max_items > 65535u) return cudaErrorInvalidValue;
    const GemmArgs a{nullptr, static_cast<const uint8_t *>(x.p), m.rows, m.rows_pad, m.panels, x.ld, 0u, out, err_flag, m.base, items, n_items};
    return tile == 64 ? gemm_experts_nt<64>(s, a, max_items, pdl) : tile == 128 ? gemm_experts_nt<128>(s, a, max_items, pdl) : cudaErrorInvalidValue;
}

}  // namespace k2t
