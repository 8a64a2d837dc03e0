// Dense (unquantized) matrices and their activations: the storage and the matrix products of the block engine
// (k2t_blocks.cu) and of kronos_cuda_linear on KRONOS_CUDA_MATRIX_DENSE matrices.
//
// bf16.  A matrix is cut into PANELS of 64 columns; a panel holds all rows (padded to 128), 128 bytes each, the eight 16-byte
// chunks of row r stored at chunk position c ^ (r % 8) - the 128-byte swizzle of the tensor-core operand layout, so ANY tile of
// 8n rows x 64 columns is one contiguous run of the image and one bulk copy puts it into shared memory as a K-major operand.
// Activations use the same form with tokens for rows (`ld` tokens per panel, a multiple of 8), written in place by the kernels
// that produce them.  Columns beyond the last are zero in the matrix and finite in the activation.
// fp32.  Row-major, rows padded to four columns (zeros); activations likewise (`ld` floats per token).
#pragma once
#include <cstdint>
#include <cuda_runtime.h>

#include "k2t_kernels.h"

namespace k2t {

constexpr Format FMT_DENSE16 = static_cast<Format>(16), FMT_DENSE32 = static_cast<Format>(17);
inline bool is_dense(const MatrixGeom &g) { return g.fmt == FMT_DENSE16 || g.fmt == FMT_DENSE32; }

constexpr uint32_t PANEL = 64;              // columns per panel
constexpr uint32_t DENSE_ROW_TILE = 128;    // rows are padded to the row tile of the tensor-core kernel
constexpr uint32_t DENSE_TOK_SLACK = 256;   // a token tile may read this many rows beyond the last panel of an activation

struct Act {                                // activation of a dense product (device memory)
    void *p;
    uint32_t ld;                            // bf16: tokens per panel; fp32: floats per token
};

inline uint32_t dense_panels(uint32_t cols) { return (cols + PANEL - 1) / PANEL; }
inline uint32_t dense_f32_ld(uint32_t cols) { return (cols + 3u) & ~3u; }
inline uint32_t act_tokens(uint32_t n_tok) { return (n_tok + 7u) & ~7u; }
inline uint32_t act_ld(bool f32, uint32_t n_tok, uint32_t cols) { return f32 ? dense_f32_ld(cols) : act_tokens(n_tok); }
inline size_t act_bytes(bool f32, uint32_t n_tok, uint32_t cols) {
    return f32 ? (size_t)n_tok * dense_f32_ld(cols) * 4 : ((size_t)dense_panels(cols) * act_tokens(n_tok) + DENSE_TOK_SLACK) * PANEL * 2;
}

struct DenseView {                          // what the kernels need of a dense matrix
    const void *base;
    uint32_t rows, cols, rows_pad, panels;  // fp32: rows_pad = floats per row
};
inline DenseView dense_view(const DeviceMatrix &m) {
    return DenseView{m.d_base, m.geom.rows, m.geom.cols, m.geom.fmt == FMT_DENSE32 ? dense_f32_ld(m.geom.cols) : m.geom.rows_pad, m.geom.nc};
}

// What becomes of the sums out[t][r] = sum over k of W[r][k] x[t][k] (fp32 accumulation).
enum class Epi : uint32_t {
    Rows,           // fp32 rows
    Softcap,        // fp32 rows of cap * tanh(sum / cap)
    Panels,         // activation of another product, column r
    Relu2,          // activation of relu(sum)^2
    GeluGated,      // rows come in pairs (gate i, up i): activation of gelu_tanh(gate) * up, column i
};
struct DenseOut {
    Epi kind;
    float *rows;                            // Rows, Softcap; scratch for the others where the matrix is fp32
    size_t stride;
    float cap;
    Act act;
};
inline DenseOut dense_rows(float *out, size_t stride) { return DenseOut{Epi::Rows, out, stride, 0.0f, Act{}}; }

// bf16: up to DENSE_TC_MIN - 1 tokens as weight passes of up to eight tokens, more on the tensor cores; fp32: plain fused
// multiply-adds, activations by a second kernel.
constexpr uint32_t DENSE_TC_MIN = 17;
cudaError_t launch_dense_out(cudaStream_t s, const DeviceMatrix &m, const Act &x, uint32_t n_tok, const DenseOut &out, int sm_count, uint32_t *err_flag,
                             uint32_t *launches, bool pdl);
inline cudaError_t launch_dense(cudaStream_t s, const DeviceMatrix &m, const Act &x, uint32_t n_tok, float *out, size_t out_stride, int sm_count,
                                uint32_t *err_flag, uint32_t *launches, bool pdl) {
    return launch_dense_out(s, m, x, n_tok, dense_rows(out, out_stride), sm_count, err_flag, launches, pdl);
}
// fp32 rows [n_tok][cols] -> activation
cudaError_t launch_dense_pack(cudaStream_t s, bool f32, const float *x, uint32_t n_tok, uint32_t cols, const Act &out, bool pdl);

// ---- one matrix per expert (all of one shape): device table of their images
struct ExpertView {
    const void *const *base;
    uint32_t rows, cols, rows_pad, panels;  // of one expert, see DenseView
};
// A stretch of rows [row0, row_end) of a packed activation that one expert works on; row0 is a multiple of eight.
struct ExpertItem { uint32_t expert, row0, row_end, pad; };
constexpr uint32_t EXPERT_TILE_MIN = 64;    // rows of the packed activation per item: 64 or 128
// tensor-core product of every item's rows (at most `tile`) with its expert; items and their number live on the device (at most max_items).
// Row p of the packed activation gives row p of the output.
cudaError_t launch_dense_experts(cudaStream_t s, const ExpertView &m, const Act &x, const ExpertItem *items, const uint32_t *n_items, uint32_t max_items,
                                 uint32_t tile, const DenseOut &out, uint32_t *err_flag, bool pdl);

}  // namespace k2t
