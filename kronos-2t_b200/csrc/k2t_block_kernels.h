// Kernels of the block engine (k2t_block_kernels.cu, k2t_window_attn.cu, k2t_delta.cu): everything between the dense products.
// `f32`: activations of the dense products are fp32 rows instead of bf16 panels (k2t_dense.h).  Residual stream, projection
// outputs and recurrent state are fp32 in both; fp32 rows have strides that are multiples of eight floats.
#pragma once
#include "k2t_dense.h"
#include "k2t_model_kernels.h"

namespace k2t {

// x[t] = table[token[t]] (bf16 table), and the same as activation
cudaError_t launch_block_embed(cudaStream_t s, bool f32, const uint16_t *table, const uint32_t *tokens, uint32_t n, float *x, size_t x_stride, const Act &out,
                               uint32_t n_tok, bool pdl);
// add: x += y / rms(y) * w, activation = x;  otherwise activation = x / rms(x) * w (x is left alone)
cudaError_t launch_block_norm(cudaStream_t s, bool f32, bool add, float *x, size_t x_stride, const float *y, size_t y_stride, const float *w, uint32_t n, float eps,
                              const Act &out, uint32_t n_tok, bool pdl);

// Per-layer token input: g = gelu_tanh(gate x) * e, x += (proj g) / rms(proj g) * w, e = table[token][offset ..]
struct SideArgs {
    DenseView gate, proj;              // [dim][n], [n][dim]
    const float *norm;                 // [n]
    const uint16_t *table;             // bf16 [vocab][table_stride]
    const uint32_t *tokens;
    uint32_t dim, table_stride, offset;
};
// short batches: residual add of the sublayer output y, and the token input, in one launch (a thread-block cluster per token)
cudaError_t launch_norm_side(cudaStream_t s, bool f32, float *x, size_t x_stride, const float *y, size_t y_stride, const float *w, uint32_t n, float eps,
                             const SideArgs &side, const Act &out, uint32_t n_tok, uint32_t *err_flag, bool pdl);
bool norm_side_fits(uint32_t n, uint32_t dim);
// prompt batches: z [n_tok][dim] = gate x is a dense product; this makes the activation of `proj`
cudaError_t launch_side_gelu(cudaStream_t s, bool f32, const float *z, size_t z_stride, const SideArgs &side, const Act &out, uint32_t n_tok, bool pdl);
// activation = a N(z) + b N(z^2) + c N(z^3) + e with (a, b, c, e) = coef, N = division by the root mean square over the n values
cudaError_t launch_polynorm(cudaStream_t s, bool f32, const float *z, size_t z_stride, uint32_t n, const float *coef, float eps, const Act &out, uint32_t n_tok, bool pdl);

// ---- sliding-window attention with per-head score scale and linear distance bias over a ring cache of unquantized rows
struct WindowAttnArgs {
    const float *qkv;                  // [n_tok][qkv_stride]: n_q x dim queries, n_kv x dim keys, n_kv x vdim values
    size_t qkv_stride;
    const float *q_norm, *k_norm;      // [dim]
    const float *head_scale, *head_slope;    // [n_q]: score = (q . k) * scale - slope * distance
    void *k_cache, *v_cache;           // [n_kv][ring rows][row] bf16 or fp32, row = window_attn_row(dim, vdim) elements, padding zero
    void *q;                           // scratch: normalised queries [n_tok][n_q][row], element type of the cache
    const uint32_t *pos;               // device: position of the first token
    uint32_t n_q, n_kv, dim, vdim, row;
    KvRing ring;                       // sinks 0; window 0 = every earlier position
    float eps;
    Act out;                           // [n_tok][n_q * vdim]
    uint32_t *err_flag;
};
bool window_attn_fits(bool f32, uint32_t group, uint32_t row);       // queries of a group beside one another in shared memory
uint32_t window_attn_row(uint32_t dim, uint32_t vdim);       // cache row in elements; 0 = larger than the kernels support
// n_tok == 1: one kernel (norms, cache row, attention); prompts: cache rows and queries, then the attention.  Returns the launches.
cudaError_t launch_window_attention(cudaStream_t s, bool f32, const WindowAttnArgs &a, uint32_t n_tok, int sm_count, uint32_t *launches, bool pdl);

// ---- generalized delta rule: S <- diag(w) S - (a u)(u^T S) + k v^T, o = S^T r; state [heads][drow][drow] fp32 (key-major)
struct DeltaArgs {
    const float *in;                   // [n_tok][in_stride]: r, k, v, g, a-logit (heads x dim each), then the decay rank's inputs
    size_t in_stride;
    DenseView decay;                   // [heads * dim][rank]
    const float *decay_bias, *rate_bias, *norm;      // [heads * dim]
    float *state;
    const float *decay_logit;          // prompts: decay product [n_tok][logit_stride]
    size_t logit_stride;
    float *rec, *o;                    // prompts, scratch: delta_record_floats(n_tok, ..), [n_tok][heads][drow]
    uint32_t heads, dim, drow, rank;
    float decay_scale, unit_eps, eps;
    Act out;                           // [n_tok][heads * dim]
    uint32_t *err_flag;
};
uint32_t delta_row(uint32_t dim);      // dim rounded up to 64; 0 = larger than the kernels support
size_t delta_record_floats(uint32_t n_tok, uint32_t heads, uint32_t drow);
bool delta_step_fits(const DeltaArgs &a);
cudaError_t launch_delta_step(cudaStream_t s, bool f32, const DeltaArgs &a, bool pdl);                                   // one token, one launch
cudaError_t launch_delta_tanh(cudaStream_t s, bool f32, const DeltaArgs &a, const Act &out, uint32_t n_tok, bool pdl);   // activation of the decay product
cudaError_t launch_delta_prompt(cudaStream_t s, bool f32, const DeltaArgs &a, uint32_t n_tok, int sm_count, bool pdl);   // three launches

}  // namespace k2t
