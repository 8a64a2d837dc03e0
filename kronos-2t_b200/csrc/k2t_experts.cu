// Router and experts of the block engine (k2t_block_kernels.h), unquantized.
//   * route_kernel: softmax over all experts and the top choices of every token, activation of the shared expert.
//   * few tokens: expert_gemv_kernel - a warp owns eight rows of an expert's matrix (or of all chosen experts' matrices, weighted
//     sum included) like the dense GEMV; the second product knows its experts before its dependency wait and asks for its first
//     panels there.
//   * prompt batches: expert_plan_kernel sorts the (token, choice) pairs by expert (counting sort, order within an expert = token
//     order, so a run repeats bit for bit), expert_gather_kernel packs the activations, the products of all experts are one
//     tensor-core launch each (launch_dense_experts), and the weighted sum rides in the residual norm (NormArgs).
#include <algorithm>

#include "k2t_block_kernels.h"
#include "k2t_dense.cuh"

namespace k2t {
namespace {

constexpr uint32_t RT_THREADS = 1024, EX_THREADS = 256, EX_PF = 8, EX_MAX_SLOTS = 33;      // top <= 32, and the shared expert

template <bool F32>
__global__ void __launch_bounds__(RT_THREADS) route_kernel(const RouteArgs a) {
    __shared__ float s[ROUTE_MAX_EXPERTS];
    const uint32_t t = blockIdx.x, tid = threadIdx.x, lane = tid & 31;
    pdl_wait();
    pdl_trigger();
    const float *z = a.z + t * a.z_stride;
    if (tid < 32) {
        float m = -INFINITY, sum = 0.0f;
        for (uint32_t e = lane; e < a.experts; e += 32) { const float v = __ldcg(z + e); s[e] = v; m = fmaxf(m, v); }
#pragma unroll
        for (int k = 16; k > 0; k >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, k));
        for (uint32_t e = lane; e < a.experts; e += 32) { const float v = expf(s[e] - m); s[e] = v; sum += v; }
        sum = warp_sum(sum);
        for (uint32_t k = 0; k < a.top; ++k) {
            float best = -1.0f;
            uint32_t id = 0xffffffffu;
            for (uint32_t e = lane; e < a.experts; e += 32)
                if (s[e] > best) { best = s[e]; id = e; }
#pragma unroll
            for (int d = 16; d > 0; d >>= 1) {
                const float ob = __shfl_xor_sync(0xffffffffu, best, d);
                const uint32_t oi = __shfl_xor_sync(0xffffffffu, id, d);
                if (ob > best || (ob == best && oi < id)) { best = ob; id = oi; }
            }
            id = min(id, a.experts - 1);          // logits that are not numbers: some expert all the same
            if (lane == 0) { a.ids[t * a.top + k] = id; a.weight[t * a.top + k] = best / sum; }
            if (lane == (id & 31u)) s[id] = -2.0f;          // the lane that reads it
        }
    } else {
        const float *h = z + a.experts;
        for (uint32_t i = tid - 32; i < a.shared_ff; i += blockDim.x - 32)
            act_store<F32>(a.shared, t, i, a.act == Epi::GeluGated ? gelu_tanh(__ldcg(h + 2 * i)) * __ldcg(h + 2 * i + 1) : relu_squared(__ldcg(h + i)));
    }
}

__device__ __forceinline__ uint32_t block_scan_1024(uint32_t v, uint32_t *s_warp, uint32_t &total) {      // exclusive
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    uint32_t x = v;
#pragma unroll
    for (uint32_t d = 1; d < 32; d <<= 1) { const uint32_t y = __shfl_up_sync(0xffffffffu, x, d); if (lane >= d) x += y; }
    __syncthreads();
    if (lane == 31) s_warp[warp] = x;
    __syncthreads();
    uint32_t before = 0;
    total = 0;
    for (uint32_t w = 0; w < 32; ++w) { if (w < warp) before += s_warp[w]; total += s_warp[w]; }
    return before + x - v;
}

// One CTA of 32 warps, warp = a stretch of the pairs; thread = expert in between.
__global__ void __launch_bounds__(1024) expert_plan_kernel(const RouteArgs a, uint32_t pairs, uint32_t tile, ExpertItem *__restrict__ items, uint32_t *__restrict__ n_items) {
    extern __shared__ uint32_t s_hist[];          // [32][experts]
    __shared__ uint32_t s_first[ROUTE_MAX_EXPERTS], s_warp[32];
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, E = a.experts;
    for (uint32_t i = tid; i < 32 * E; i += 1024) s_hist[i] = 0;
    pdl_wait();
    pdl_trigger();
    __syncthreads();
    const uint32_t per = ((pairs + 1023) / 1024) * 32, p0 = warp * per, p1 = min(pairs, p0 + per);
    uint32_t *hist = s_hist + warp * E;
    constexpr uint32_t AHEAD = 4;          // ids of the next steps are on their way
    for (uint32_t p = p0; p < p1; p += 32 * AHEAD) {
        uint32_t id[AHEAD];
#pragma unroll
        for (uint32_t i = 0; i < AHEAD; ++i) id[i] = p + 32 * i + lane < p1 ? __ldcg(a.ids + p + 32 * i + lane) : 0u;
#pragma unroll
        for (uint32_t i = 0; i < AHEAD; ++i) {
            const uint32_t q = p + 32 * i + lane;
            const bool in = q < p1;
            const uint32_t active = __ballot_sync(0xffffffffu, in);
            if (in) {
                const uint32_t same = __match_any_sync(active, id[i]), rank = __popc(same & ((1u << lane) - 1u)), base = hist[id[i]];
                __syncwarp(active);
                if (rank == 0) hist[id[i]] = base + __popc(same);
                a.row[q] = base + rank;
            }
            __syncwarp();
        }
    }
    __syncthreads();
    uint32_t count = 0;
    if (tid < E)
        for (uint32_t w = 0; w < 32; ++w) { const uint32_t c = s_hist[w * E + tid]; s_hist[w * E + tid] = count; count += c; }
    uint32_t total_rows, total_items;
    const uint32_t first = block_scan_1024((count + 7u) & ~7u, s_warp, total_rows), n = (count + tile - 1) / tile;
    const uint32_t at = block_scan_1024(n, s_warp, total_items);
    if (tid < E) {
        s_first[tid] = first;
        for (uint32_t i = 0; i < n; ++i) items[at + i] = ExpertItem{tid, first + i * tile, min(first + count, first + (i + 1) * tile), 0u};
    }
    if (tid == 0) *n_items = total_items;
    __syncthreads();
#pragma unroll 4
    for (uint32_t p = p0 + lane; p < p1; p += 32) {
        const uint32_t e = __ldcg(a.ids + p);
        a.row[p] += s_first[e] + hist[e];
    }
}

__global__ void __launch_bounds__(256) expert_gather_kernel(const RouteArgs a, const Act x, uint32_t panels, const Act out, uint32_t pairs) {
    pdl_wait();
    pdl_trigger();
    const uint32_t per = panels * 8;
    const uint4 *src = static_cast<const uint4 *>(x.p);
    uint4 *dst = static_cast<uint4 *>(out.p);
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < (size_t)pairs * per; i += (size_t)gridDim.x * 256) {
        const uint32_t pair = (uint32_t)(i / per), k = (uint32_t)(i % per), p = k >> 3, c = k & 7u, t = pair / a.top, r = __ldcg(a.row + pair);
        dst[((size_t)p * out.ld + r) * 8 + (c ^ (r & 7u))] = __ldcg(src + ((size_t)p * x.ld + t) * 8 + (c ^ (t & 7u)));
    }
}

struct ExpertGemvArgs {
    RouteArgs route;
    ExpertView m;
    DenseView shared;                 // DOWN: second product of the shared expert (base null: none)
    Act x, out;
    float *rows;                      // DOWN
    size_t stride;
    uint32_t wk_log2;
};

// UP: blockIdx.y = choice k of token blockIdx.z.  DOWN: all choices of token blockIdx.z, their panels one after the other.
template <bool DOWN>
__global__ void __launch_bounds__(EX_THREADS, 2) expert_gemv_kernel(const ExpertGemvArgs a) {
    __shared__ float s_part[8][8], s_w[EX_MAX_SLOTS];
    __shared__ const uint4 *s_base[EX_MAX_SLOTS];
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, wk = 1u << a.wk_log2, c = lane & 7u, r = lane >> 3, t = blockIdx.z, top = a.route.top;
    const uint32_t group = blockIdx.x * (8u >> a.wk_log2) + (warp >> a.wk_log2), ks = warp & (wk - 1);
    const bool live = group * 8 < a.m.rows;
    const uint32_t np = a.m.panels, n_exp = DOWN ? top : 1u, total = n_exp * np + (DOWN && a.shared.base != nullptr ? a.shared.panels : 0u);
    if (!DOWN) { pdl_wait(); pdl_trigger(); }          // the second product's choices were made two kernels ago
    if (tid < n_exp) {
        const uint32_t i = t * top + (DOWN ? tid : blockIdx.y);
        s_base[tid] = static_cast<const uint4 *>(a.m.base[__ldcg(a.route.ids + i)]);
        s_w[tid] = DOWN ? __ldcg(a.route.weight + i) : 1.0f;
    }
    if (DOWN && tid == n_exp) { s_base[tid] = static_cast<const uint4 *>(a.shared.base); s_w[tid] = 1.0f; }
    __syncthreads();
    // position f of the concatenated panels: (matrix, panel, pitch of its panels)
    auto weights = [&](uint32_t f, uint4 &u, uint4 &v) {
        const uint32_t slot = min(f / np, n_exp), p = f - slot * np;
        const uint4 *w = s_base[slot] + (size_t)p * (DOWN && slot == n_exp ? a.shared.rows_pad : a.m.rows_pad) * 8 + group * 64;
        u = ldg_stream(w + r * 8 + (c ^ r));
        v = ldg_stream(w + (r + 4) * 8 + (c ^ (r + 4)));
    };
    uint4 u[EX_PF], v[EX_PF];
#pragma unroll
    for (uint32_t i = 0; i < EX_PF; ++i)
        if (live && ks + i * wk < total) weights(ks + i * wk, u[i], v[i]);
    if (DOWN) { pdl_wait(); pdl_trigger(); }
    float acc0 = 0.0f, acc1 = 0.0f;
    if (live)
        for (uint32_t f0 = ks; f0 < total; f0 += EX_PF * wk)
#pragma unroll
            for (uint32_t i = 0; i < EX_PF; ++i) {
                const uint32_t f = f0 + i * wk;
                if (f >= total) break;
                const uint32_t slot = min(f / np, n_exp), p = f - slot * np;
                const bool sh = DOWN && slot == n_exp;
                const Act &x = sh ? a.route.shared : a.x;
                const uint32_t row = !DOWN || sh ? t : t * top + slot;
                const uint4 q = __ldcg(static_cast<const uint4 *>(x.p) + ((size_t)p * x.ld + row) * 8 + (c ^ (row & 7u)));
                const float4 lo = make_float4(bf_lo(q.x), bf_hi(q.x), bf_lo(q.y), bf_hi(q.y)), hi = make_float4(bf_lo(q.z), bf_hi(q.z), bf_lo(q.w), bf_hi(q.w));
                __align__(16) const float xs[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
                const float d0 = dot8(u[i], xs, 0.0f), d1 = dot8(v[i], xs, 0.0f), w = s_w[slot];
                acc0 = __fmaf_rn(w, d0, acc0);
                acc1 = __fmaf_rn(w, d1, acc1);
                if (f + EX_PF * wk < total) weights(f + EX_PF * wk, u[i], v[i]);
            }
#pragma unroll
    for (int m = 1; m < 8; m <<= 1) {
        acc0 = __fadd_rn(acc0, __shfl_xor_sync(0xffffffffu, acc0, m));
        acc1 = __fadd_rn(acc1, __shfl_xor_sync(0xffffffffu, acc1, m));
    }
    if (c == 0) { s_part[warp][r] = acc0; s_part[warp][r + 4] = acc1; }
    __syncthreads();
    const uint32_t groups = 8u >> a.wk_log2;
    if (tid < groups * 8) {
        const uint32_t row_l = tid & 7u, g = tid >> 3, row = (blockIdx.x * groups + g) * 8 + row_l;
        if (row >= a.m.rows) return;
        float s = 0.0f, s1 = 0.0f;
        for (uint32_t k = 0; k < wk; ++k) s = __fadd_rn(s, s_part[g * wk + k][row_l]);
        if (DOWN) {
            a.rows[(size_t)t * a.stride + row] = s;
        } else {
            if ((row_l & 1u) == 0)
                for (uint32_t k = 0; k < wk; ++k) s1 = __fadd_rn(s1, s_part[g * wk + k][row_l + 1]);
            dense_store<false>(DenseOut{a.route.act, nullptr, 0, 0.0f, a.out}, t * top + blockIdx.y, row, s, s1);
        }
    }
}

__device__ __forceinline__ float row_dot_f32(const float *w, const float *x, uint32_t cols, uint32_t lane) {
    float s = 0.0f;
    for (uint32_t k = lane; k < cols; k += 32) s = __fmaf_rn(__ldg(w + k), __ldcg(x + k), s);
    return warp_sum(s);
}

// fp32 forms, one warp per row (UP: per output column); grid.y = (token, choice) or token
template <bool DOWN>
__global__ void __launch_bounds__(EX_THREADS) expert_gemv_f32_kernel(const ExpertGemvArgs a) {
    const uint32_t lane = threadIdx.x & 31, o = blockIdx.x * 8 + (threadIdx.x >> 5), t = blockIdx.z, top = a.route.top;
    pdl_wait();
    pdl_trigger();
    const bool gated = a.route.act == Epi::GeluGated;
    if (o >= (DOWN || !gated ? a.m.rows : a.m.rows / 2)) return;
    const float *x = static_cast<const float *>(a.x.p);
    if (DOWN) {
        float y = 0.0f;
        for (uint32_t k = 0; k < top; ++k) {
            const uint32_t i = t * top + k;
            const float d = row_dot_f32(static_cast<const float *>(a.m.base[__ldcg(a.route.ids + i)]) + (size_t)o * a.m.rows_pad, x + (size_t)i * a.x.ld, a.m.cols, lane);
            y = __fmaf_rn(__ldcg(a.route.weight + i), d, y);
        }
        if (a.shared.base != nullptr)
            y += row_dot_f32(static_cast<const float *>(a.shared.base) + (size_t)o * a.shared.rows_pad, static_cast<const float *>(a.route.shared.p) + (size_t)t * a.route.shared.ld, a.shared.cols, lane);
        if (lane == 0) a.rows[(size_t)t * a.stride + o] = y;
    } else {
        const uint32_t i = t * top + blockIdx.y;
        const float *w = static_cast<const float *>(a.m.base[__ldcg(a.route.ids + i)]), *xr = x + (size_t)t * a.x.ld;
        const float d = row_dot_f32(w + (size_t)(gated ? 2 * o : o) * a.m.rows_pad, xr, a.m.cols, lane);
        const float v = gated ? gelu_tanh(d) * row_dot_f32(w + (size_t)(2 * o + 1) * a.m.rows_pad, xr, a.m.cols, lane) : relu_squared(d);
        if (lane == 0) act_store<true>(a.out, i, o, v);
    }
}

// warps per row group: about one wave of CTAs, but a handful of panels per warp at least
uint32_t split_warps(uint32_t groups, uint32_t panels, int sm_count) {
    uint32_t wl = 0;
    while (wl < 3 && (2u << wl) * 4 <= panels && groups << wl <= 8u * (uint32_t)sm_count) ++wl;
    return wl;
}

}  // namespace

cudaError_t launch_route(cudaStream_t s, bool f32, const RouteArgs &a, uint32_t n_tok, bool pdl) {
    const uint32_t threads = n_tok > 64 ? 256u : std::min(RT_THREADS, 64u + ((a.shared_ff + 31u) & ~31u));
    return launch_kernel(f32 ? route_kernel<true> : route_kernel<false>, dim3(n_tok), dim3(threads), 0, s, pdl, a);
}

uint32_t expert_rows(uint32_t n_tok, uint32_t top, uint32_t experts) { return (n_tok * top + 7 * std::min(experts, n_tok * top) + 7u) & ~7u; }
uint32_t expert_tile(uint32_t n_tok, uint32_t top, uint32_t experts) {
    const uint32_t share = n_tok * top / experts;
    return share >= 96 ? 128u : EXPERT_TILE_MIN;
}
uint32_t expert_items(uint32_t n_tok, uint32_t top, uint32_t experts) { return n_tok * top / expert_tile(n_tok, top, experts) + std::min(experts, n_tok * top); }

cudaError_t launch_expert_plan(cudaStream_t s, const RouteArgs &a, uint32_t n_tok, ExpertItem *items, uint32_t *n_items, bool pdl) {
    const size_t smem = (size_t)32 * a.experts * 4;
    cudaError_t e = allow_dynamic_smem(reinterpret_cast<const void *>(expert_plan_kernel), smem);
    if (e != cudaSuccess) return e;
    return launch_kernel(expert_plan_kernel, dim3(1), dim3(1024), smem, s, pdl, a, n_tok * a.top, expert_tile(n_tok, a.top, a.experts), items, n_items);
}

cudaError_t launch_expert_gather(cudaStream_t s, const RouteArgs &a, const Act &x, uint32_t cols, const Act &out, uint32_t n_tok, bool pdl) {
    const uint32_t panels = dense_panels(cols), pairs = n_tok * a.top;
    const uint32_t ctas = (uint32_t)std::min<size_t>(2368, ((size_t)pairs * panels * 8 + 255) / 256);
    return launch_kernel(expert_gather_kernel, dim3(ctas), dim3(256), 0, s, pdl, a, x, panels, out, pairs);
}

cudaError_t launch_expert_up(cudaStream_t s, bool f32, const RouteArgs &a, const ExpertView &m, const Act &x, const Act &out, uint32_t n_tok, int sm_count, bool pdl) {
    if (a.top + 1 > EX_MAX_SLOTS || n_tok > 65535u) return cudaErrorInvalidValue;
    ExpertGemvArgs g{a, m, DenseView{}, x, out, nullptr, 0, 0};
    if (f32) return launch_kernel(expert_gemv_f32_kernel<false>, dim3((m.rows + 7) / 8, a.top, n_tok), dim3(EX_THREADS), 0, s, pdl, g);
    const uint32_t groups = (m.rows + 7) / 8;
    g.wk_log2 = split_warps(groups * a.top * n_tok, m.panels, sm_count);
    const uint32_t per = 8u >> g.wk_log2;
    return launch_kernel(expert_gemv_kernel<false>, dim3((groups + per - 1) / per, a.top, n_tok), dim3(EX_THREADS), 0, s, pdl, g);
}

cudaError_t launch_expert_down(cudaStream_t s, bool f32, const RouteArgs &a, const ExpertView &m, const Act &x, const DenseView &shared_down, float *out,
                               size_t out_stride, uint32_t n_tok, int sm_count, bool pdl) {
    if (a.top + 1 > EX_MAX_SLOTS || n_tok > 65535u) return cudaErrorInvalidValue;
    ExpertGemvArgs g{a, m, shared_down, x, Act{}, out, out_stride, 0};
    if (f32) return launch_kernel(expert_gemv_f32_kernel<true>, dim3((m.rows + 7) / 8, 1, n_tok), dim3(EX_THREADS), 0, s, pdl, g);
    const uint32_t groups = (m.rows + 7) / 8;
    g.wk_log2 = split_warps(groups * n_tok, m.panels * a.top + (shared_down.base ? shared_down.panels : 0), sm_count);
    const uint32_t per = 8u >> g.wk_log2;
    return launch_kernel(expert_gemv_kernel<true>, dim3((groups + per - 1) / per, 1, n_tok), dim3(EX_THREADS), 0, s, pdl, g);
}

}  // namespace k2t
