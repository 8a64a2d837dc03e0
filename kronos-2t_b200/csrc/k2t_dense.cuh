// Device side of the dense storage (k2t_dense.h): element addressing, short row products, cluster reductions.
#pragma once
#include <cuda_bf16.h>

#include "k2t_dense.h"
#include "k2t_device.cuh"

namespace k2t {

__device__ __forceinline__ size_t panel_index(uint32_t ld, uint32_t row, uint32_t k) {      // in elements
    return ((size_t)(k >> 6) * ld + row) * PANEL + ((((k >> 3) & 7u) ^ (row & 7u)) << 3) + (k & 7u);
}
template <bool F32> __device__ __forceinline__ void act_store(const Act &a, uint32_t t, uint32_t k, float v) {
    if (F32) static_cast<float *>(a.p)[(size_t)t * a.ld + k] = v;
    else static_cast<__nv_bfloat16 *>(a.p)[panel_index(a.ld, t, k)] = __float2bfloat16_rn(v);
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t *>(&v);
}
// columns k .. k+3 (k a multiple of 4); columns at and beyond n are not written
template <bool F32> __device__ __forceinline__ void act_store4(const Act &a, uint32_t t, uint32_t k, uint32_t n, float4 v) {
    if (k + 4 <= n) {
        if (F32) *reinterpret_cast<float4 *>(static_cast<float *>(a.p) + (size_t)t * a.ld + k) = v;
        else *reinterpret_cast<uint2 *>(static_cast<__nv_bfloat16 *>(a.p) + panel_index(a.ld, t, k)) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
    } else {
        const float e[4] = {v.x, v.y, v.z, v.w};
        for (uint32_t i = 0; i < 4 && k + i < n; ++i) act_store<F32>(a, t, k + i, e[i]);
    }
}
__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xFFFF0000u); }
// eight consecutive fp32 values (shared or global memory, 16-byte aligned) times a 16-byte chunk of bf16 weights
__device__ __forceinline__ float dot8(const uint4 &w, const float *x, float acc) {
    const float4 a = *reinterpret_cast<const float4 *>(x), b = *reinterpret_cast<const float4 *>(x + 4);
    acc = __fmaf_rn(bf_lo(w.x), a.x, acc); acc = __fmaf_rn(bf_hi(w.x), a.y, acc);
    acc = __fmaf_rn(bf_lo(w.y), a.z, acc); acc = __fmaf_rn(bf_hi(w.y), a.w, acc);
    acc = __fmaf_rn(bf_lo(w.z), b.x, acc); acc = __fmaf_rn(bf_hi(w.z), b.y, acc);
    acc = __fmaf_rn(bf_lo(w.w), b.z, acc); acc = __fmaf_rn(bf_hi(w.w), b.w, acc);
    return acc;
}
// Product of matrix row `row`, panels [p0, p1), with x (shared memory; x[0] belongs to column 64 p0, zero beyond the last
// column) by eight consecutive lanes (sub = lane % 8); every one of them receives the sum.  SHARED: the panels were copied to
// shared memory.
template <bool F32, bool SHARED = false> __device__ __forceinline__ float row_dot8(const DenseView &m, uint32_t row, uint32_t p0, uint32_t p1, const float *x, uint32_t sub) {
    float acc = 0.0f;
    if (F32) {
        const float *w = static_cast<const float *>(m.base) + (size_t)row * m.rows_pad;
        const uint32_t k1 = min(p1 * PANEL, m.cols);
        for (uint32_t k = p0 * PANEL + sub; k < k1; k += 8) acc = __fmaf_rn(__ldg(w + k), x[k - p0 * PANEL], acc);
    } else {
        const uint4 *w = static_cast<const uint4 *>(m.base);
#pragma unroll SHARED ? 1 : 4
        for (uint32_t p = p0; p < p1; ++p) {
            const uint4 *q = w + ((size_t)p * m.rows_pad + row) * 8 + (sub ^ (row & 7u));
            acc = dot8(SHARED ? *q : __ldg(q), x + (p - p0) * PANEL + sub * 8, acc);
        }
    }
    acc = __fadd_rn(acc, __shfl_xor_sync(0xffffffffu, acc, 1));
    acc = __fadd_rn(acc, __shfl_xor_sync(0xffffffffu, acc, 2));
    acc = __fadd_rn(acc, __shfl_xor_sync(0xffffffffu, acc, 4));
    return acc;
}

// z (1 + tanh(u)) / 2 = z / (1 + exp(-2 u)): the second form keeps its relative accuracy where tanh is near -1
__device__ __forceinline__ float gelu_tanh(float z) {
    return z / (1.0f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}
// the same to bf16 accuracy and better, for values that are rounded to bf16 next
__device__ __forceinline__ float gelu_tanh_fast(float z) {
    return __fdividef(z, 1.0f + __expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float relu_squared(float z) { const float r = fmaxf(z, 0.0f); return r * r; }
__device__ __forceinline__ float softcap(float z, float cap) { return cap * tanhf(z / cap); }
// sum of row r (and, for pairs, of row r + 1 behind an even r) of token t -> output
template <bool F32> __device__ __forceinline__ void dense_store(const DenseOut &o, uint32_t t, uint32_t r, float v, float next) {
    switch (o.kind) {
        case Epi::Rows: o.rows[(size_t)t * o.stride + r] = v; break;
        case Epi::Softcap: o.rows[(size_t)t * o.stride + r] = softcap(v, o.cap); break;
        case Epi::Panels: act_store<F32>(o.act, t, r, v); break;
        case Epi::Relu2: act_store<F32>(o.act, t, r, relu_squared(v)); break;
        case Epi::GeluGated:
            if ((r & 1u) == 0) act_store<F32>(o.act, t, r >> 1, gelu_tanh(v) * next);
            break;
    }
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int m = 16; m > 0; m >>= 1) v = __fadd_rn(v, __shfl_xor_sync(0xffffffffu, v, m));
    return v;
}
// Sum over the CTA (blockDim.x a multiple of 32, at most 1024) of N values per thread; every thread receives the sums.
// scratch: 32 * N floats of shared memory, free again when the next __syncthreads has passed.
template <int N> __device__ __forceinline__ void block_sum(float (&v)[N], float *scratch) {
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = warp_sum(v[i]);
    __syncthreads();
    if (lane == 0)
#pragma unroll
        for (int i = 0; i < N; ++i) scratch[warp * N + i] = v[i];
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = warp_sum(lane < nw ? scratch[lane * N + i] : 0.0f);
}

// ---- thread-block clusters
__device__ __forceinline__ uint32_t cluster_rank() { uint32_t r; asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ uint32_t cluster_size() { uint32_t r; asm volatile("mov.u32 %0, %%cluster_nctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ void st_cluster_f32(const float *local, uint32_t rank, float v) {      // the same shared-memory word of CTA `rank`
    uint32_t dst;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dst) : "r"((uint32_t)__cvta_generic_to_shared(local)), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(v) : "memory");
}
__device__ __forceinline__ float ld_cluster_f32(const float *local, uint32_t rank) {
    uint32_t src;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(src) : "r"((uint32_t)__cvta_generic_to_shared(local)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(src) : "memory");
    return v;
}
// Sum over the cluster of N values every thread of a CTA already holds alike (block_sum); added in rank order, so all CTAs
// get the same bits.  slots: cluster_size * N floats of shared memory, written by the peers: one use per kernel and slot array.
template <int N> __device__ __forceinline__ void cluster_sum(float (&v)[N], float *slots) {
    const uint32_t cs = cluster_size(), me = cluster_rank();
    if (cs == 1) return;
    if (threadIdx.x < cs)
#pragma unroll
        for (int i = 0; i < N; ++i) st_cluster_f32(slots + me * N + i, threadIdx.x, v[i]);
    cluster_sync_all();
#pragma unroll
    for (int i = 0; i < N; ++i) {
        float s = 0.0f;
        for (uint32_t r = 0; r < cs; ++r) s = __fadd_rn(s, slots[r * N + i]);
        v[i] = s;
    }
}

// Launches `kernel` as clusters of `cs` CTAs along x, optionally as a programmatic dependent (see launch_kernel).
template <typename... KArgs, typename... Args>
inline cudaError_t launch_cluster(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, bool pdl, uint32_t cs, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = cs; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr; cfg.numAttrs = pdl ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

}  // namespace k2t
