// Kernels of the block engine (k2t_block_kernels.cu, k2t_window_attn.cu, k2t_delta.cu, k2t_latent_attn.cu, k2t_experts.cu): everything between the dense products.
// `f32`: activations of the dense products are fp32 rows instead of bf16 panels (k2t_dense.h).  Residual stream, projection
// outputs and recurrent state are fp32 in both; fp32 rows have strides that are multiples of eight floats.
#pragma once
#include "k2t_dense.h"
#include "k2t_model_kernels.h"

namespace k2t {

// x[t] = table[token[t]] (bf16 table), and the same as activation
cudaError_t launch_block_embed(cudaStream_t s, bool f32, const uint16_t *table, const uint32_t *tokens, uint32_t n, float *x, size_t x_stride, const Act &out,
                               uint32_t n_tok, bool pdl);
// Residual step and the norm in front of the next sublayer, rms(v) = sqrt(mean(v^2) + eps):
//   y (when given): x += mult * y / rms(y) * post;   activation = x / rms(x) * pre, or x without `pre`.
// With `top`, y[t] first receives the sum over k of weight[t][k] * pairs[row[t][k]]: the outputs of a token's experts.
struct NormArgs {
    float *x;
    size_t x_stride;
    float *y;
    size_t y_stride;
    const float *post, *pre;
    float mult, eps;
    uint32_t n, top;
    const float *pairs, *weight;       // [rows][pair_stride], [n_tok][top]
    size_t pair_stride;
    const uint32_t *row;               // [n_tok][top]
    Act out;
};
cudaError_t launch_block_norm(cudaStream_t s, bool f32, const NormArgs &a, uint32_t n_tok, bool pdl);

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


// ---- latent attention: queries and keys through low-rank latents; a position caches its key/value latent c and one rotated key
// part shared by all heads.  score = (q . (W_uk c) + q_rot . k_rot) * scale, value = W_uv c.
//   * Few tokens (and fp32): q is brought into latent space (W_uk^T q), attention runs over the cached rows themselves in splits of
//     the positions, the sums over c go through W_uv when the splits are merged.
//   * Prompt batches (bf16): keys and values of every head are expanded by one product over the cached rows, then a
//     tensor-core attention kernel (tcgen05, scores and sums in tensor memory) runs per head and 128 tokens.
struct LatentShape {
    uint32_t heads, dim, rot_dim, vdim, q_rank, kv_rank;
    // all that follows is in elements of 64-column panels (fp32: kv_rank and rot_dim rounded up to four columns)
    uint32_t rot_at;                   // column of the rotated part in a cached row (and of the rotated query part)
    uint32_t row;                      // columns of a cached row
};
LatentShape latent_shape(bool f32, uint32_t heads, uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t q_rank, uint32_t kv_rank);
#ifdef __CUDACC__
__host__ __device__
#endif
inline uint32_t latent_head_cols(uint32_t dim) { return (dim + 63u) & ~63u; }      // rows of a head in kv_up (and columns of the expanded forms)
bool latent_attn_fits(bool f32, const LatentShape &d);
bool latent_flash_fits(const LatentShape &d);
constexpr uint32_t LATENT_TOKENS = 128;      // most tokens of one launch over the cached rows

struct LatentAttnArgs {
    LatentShape d;
    const float *in;                   // [n_tok][in_stride]: query latent, key/value latent, rotated key part
    size_t in_stride;
    const float *q, *q_norm, *kv_norm; // q: [n_tok][q_stride] heads x (dim, rot_dim)
    size_t q_stride;
    const float *rot;                  // [positions][rot_dim]: (cos, sin) of every pair
    DenseView kv_up;                   // [heads * head_cols(dim) + heads * head_cols(vdim)][kv_rank]
    Act cache;                         // one row per position; bf16: `ld` positions (a multiple of 128) per panel
    const uint32_t *pos;               // device: position of the first token
    float scale, eps;
    Act q_lat;                         // activation of the query product [n_tok][q_rank]
    Act q_rows;                        // few tokens: [n_tok * heads][row];  prompts: [n_tok][heads * (head_cols(dim) + head_cols(rot_dim))]
    Act kv;                            // prompts: expanded keys, then values, of all positions seen
    float *part_o, *part_m, *part_l;   // few tokens: [n_tok * heads][splits][kv_rank rounded up to four], [..][splits]
    Act out;                           // [n_tok][heads * vdim]
    uint32_t *err_flag;
};
// query latent and cache row of every token (norms, rotation)
cudaError_t launch_latent_prep(cudaStream_t s, bool f32, const LatentAttnArgs &a, uint32_t n_tok, bool pdl);
uint32_t latent_splits(const LatentShape &d, uint32_t n_tok, uint32_t max_positions, int sm_count);
// tokens t0 .. t0 + n_tok - 1 of the batch (at most LATENT_TOKENS), three launches
cudaError_t launch_latent_few(cudaStream_t s, bool f32, const LatentAttnArgs &a, uint32_t t0, uint32_t n_tok, uint32_t splits, bool pdl);
// prompt batch, two launches; `kv` has been filled
cudaError_t launch_latent_prompt(cudaStream_t s, const LatentAttnArgs &a, uint32_t n_tok, bool pdl);

// ---- router and experts: softmax over the logits of all experts, the `top` largest (lower index first), weights = their scores
struct RouteArgs {
    const float *z;                    // [n_tok][z_stride]: expert logits, then the rows of the shared expert's first product
    size_t z_stride;
    uint32_t experts, top;
    uint32_t *ids, *row;               // [n_tok][top]; row: place in the packed activation, set by launch_expert_plan
    float *weight;
    Epi act;                           // Relu2 or GeluGated
    uint32_t shared_ff;                // 0: no shared expert
    Act shared;                        // activation of its second product
};
cudaError_t launch_route(cudaStream_t s, bool f32, const RouteArgs &a, uint32_t n_tok, bool pdl);
constexpr uint32_t ROUTE_MAX_EXPERTS = 1024;
// packed rows of a batch: (token, k) pairs sorted by expert, every expert's stretch starting at a multiple of eight
uint32_t expert_rows(uint32_t n_tok, uint32_t top, uint32_t experts);
uint32_t expert_tile(uint32_t n_tok, uint32_t top, uint32_t experts);          // rows per item: most experts' shares in few items
uint32_t expert_items(uint32_t n_tok, uint32_t top, uint32_t experts);
cudaError_t launch_expert_plan(cudaStream_t s, const RouteArgs &a, uint32_t n_tok, ExpertItem *items, uint32_t *n_items, bool pdl);
cudaError_t launch_expert_gather(cudaStream_t s, const RouteArgs &a, const Act &x, uint32_t cols, const Act &out, uint32_t n_tok, bool pdl);
// few tokens: every pair against its expert's matrix.  up: activation row t * top + k.  down: y[t] = sum over k of weight * (down h)
// + the shared expert's product, fp32 rows
cudaError_t launch_expert_up(cudaStream_t s, bool f32, const RouteArgs &a, const ExpertView &m, const Act &x, const Act &out, uint32_t n_tok, int sm_count, bool pdl);
cudaError_t launch_expert_down(cudaStream_t s, bool f32, const RouteArgs &a, const ExpertView &m, const Act &x, const DenseView &shared_down, float *out,
                               size_t out_stride, uint32_t n_tok, int sm_count, bool pdl);

}  // namespace k2t
