// Models described block by block: every block names its token mixer (sliding-window attention, the generalized delta rule or latent
// attention), its feed-forward (dense, experts, or none) and its sizes, over unquantized matrices.  Residual with norms behind and
// optionally in front of every sublayer: x += m norm1(mixer(pre1(x))), x += m norm2(ff(pre2(x))), then the optional per-layer token
// input.  The engine around it - graphs, prompt batches, greedy loop, argmax, launch counting, profiling - is k2t_engine.cu's; here
// are creation, the state manager (a key/value ring or a latent cache per attention layer, a state matrix per head of a recurrent
// layer, the sequence's position) and the launches of a batch.
//
// One decoded token: window-attention block = in-projection, attention (norms, cache row, softmax, one cluster launch),
// out-projection, residual norm, up, activation, down, residual norm + token input (one cluster launch); recurrent block without
// feed-forward = in-projection, recurrence (one launch), out-projection, residual norm + token input; latent-attention block =
// in-projection, latent norms + cache row, query product, queries into latent space, attention over the cached rows, merge + values,
// out-projection, residual norm + norm, up with activation, down, residual norm + norm; with experts: router and first product of the
// shared expert, choice, up of the chosen experts, their weighted down, residual norm + norm.
#include <cmath>
#include <cstdlib>
#include <cstring>
#include <map>
#include <new>

#include "k2t_block_kernels.h"
#include "k2t_blocks.h"

namespace k2t {

struct Block {
    uint32_t mixer = 0, heads = 0, kv_heads = 0, dim = 0, vdim = 0, row = 0, rank = 0, ff = 0;
    float decay_scale = 0.0f, unit_eps = 0.0f;
    float *norm1 = nullptr, *norm2 = nullptr, *q_norm = nullptr, *k_norm = nullptr, *head_scale = nullptr, *head_slope = nullptr;
    float *decay_bias = nullptr, *rate_bias = nullptr, *out_norm = nullptr, *coef = nullptr, *side_norm = nullptr;
    KronosCudaMatrix *in = nullptr, *decay = nullptr, *o = nullptr, *up = nullptr, *down = nullptr, *side_gate = nullptr, *side_proj = nullptr;
    // latent attention
    LatentShape lat{};
    bool flash = false;                        // the prompt kernel takes these sizes
    float score_scale = 0.0f;
    float *q_latent_norm = nullptr, *kv_latent_norm = nullptr, *rot = nullptr;
    KronosCudaMatrix *q_up = nullptr, *kv_up = nullptr;
    // norms in front of the sublayers; feed-forward
    float *pre1 = nullptr, *pre2 = nullptr;
    uint32_t act = 0, experts = 0, top = 0, shared_ff = 0;
    KronosCudaMatrix *router = nullptr, *shared_down = nullptr;
    std::vector<KronosCudaMatrix *> expert_up, expert_down;
    const void **d_up = nullptr, **d_down = nullptr;          // device tables of the experts' images
    // window attention: ring of key and value rows; latent attention: k = latent rows; recurrent: state [heads][row][row]
    KvRing ring{};
    uint8_t *k = nullptr, *v = nullptr;
    size_t k_bytes = 0, v_bytes = 0;
    float *state = nullptr;
    size_t state_floats = 0;
};

struct BlockModel {
    bool f32 = false, recurrent = false, windowed = false;
    float residual_mult = 1.0f, softcap = 0.0f;
    uint32_t side_dim = 0, hs = 0;             // hs: stride of fp32 hidden-sized rows
    std::vector<Block> blocks;
    KronosCudaMatrix *head = nullptr;
    float *final_norm = nullptr;
    uint16_t *embed = nullptr, *side_embed = nullptr;
    // workspace, max_batch tokens
    float *x = nullptr, *z = nullptr, *proj = nullptr, *logit = nullptr, *rec = nullptr, *scan_o = nullptr;
    void *act_x = nullptr, *act_m = nullptr, *act_s = nullptr, *q = nullptr;
    size_t zs = 0, ls = 0;                     // strides of z and of the decay logits
    // latent attention: query rows, expanded keys and values, partial results of the splits; experts: see RouteArgs
    void *act_q = nullptr, *act_kv = nullptr, *act_p = nullptr, *act_e = nullptr;
    float *part_o = nullptr, *part_m = nullptr, *part_l = nullptr, *route_w = nullptr, *pairs = nullptr;
    uint32_t *route_ids = nullptr, *route_row = nullptr, *n_items = nullptr;
    ExpertItem *items = nullptr;
    std::vector<float *> parked;               // copies of the recurrent states
    size_t pos = 0;                            // where the sequence stands
    uint32_t step_launches = 0;
};

namespace {

constexpr size_t LOST = ~(size_t)0;
constexpr uint32_t pad8(uint32_t n) { return (n + 7u) & ~7u; }

Act act_of(const BlockModel &b, void *p, uint32_t T, uint32_t cols) { return Act{p, act_ld(b.f32, T, cols)}; }

bool product_out(KronosCudaEngine *e, const KronosCudaMatrix *m, const Act &x, uint32_t T, const DenseOut &out, const char *what) {
    uint32_t n = 0;
    const cudaError_t err = launch_dense_out(e->ctx->stream, m->dm, x, T, out, e->ctx->sm_count, e->ctx->d_err, &n, e->pdl);
    return engine_count(e, err, what, n);
}
bool product(KronosCudaEngine *e, const KronosCudaMatrix *m, const Act &x, uint32_t T, float *out, size_t stride, const char *what) {
    return product_out(e, m, x, T, dense_rows(out, stride), what);
}
// activation of the next product; z serves as scratch of the fp32 form
bool product_act(KronosCudaEngine *e, const KronosCudaMatrix *m, const Act &x, uint32_t T, Epi kind, const Act &out, const char *what) {
    return product_out(e, m, x, T, DenseOut{kind, e->blocks->z, e->blocks->zs, 0.0f, out}, what);
}
Epi epi_of(uint32_t act) { return act == KRONOS_CUDA_ACT_GELU_GATED ? Epi::GeluGated : Epi::Relu2; }
uint32_t up_rows(uint32_t act, uint32_t ff) { return act == KRONOS_CUDA_ACT_GELU_GATED ? 2 * ff : ff; }

SideArgs side_args(const KronosCudaEngine *e, size_t l) {
    const BlockModel &b = *e->blocks;
    const Block &B = b.blocks[l];
    return SideArgs{dense_view(B.side_gate->dm), dense_view(B.side_proj->dm), B.side_norm, b.side_embed, e->d_token, b.side_dim,
                    b.side_dim * (uint32_t)b.blocks.size(), b.side_dim * (uint32_t)l};
}

bool mix_attention(KronosCudaEngine *e, Block &B, uint32_t T, const Act &out) {
    BlockModel &b = *e->blocks;
    WindowAttnArgs a{};
    a.qkv = b.z; a.qkv_stride = b.zs;
    a.q_norm = B.q_norm; a.k_norm = B.k_norm; a.head_scale = B.head_scale; a.head_slope = B.head_slope;
    a.k_cache = B.k; a.v_cache = B.v; a.q = b.q; a.pos = e->d_pos;
    a.n_q = B.heads; a.n_kv = B.kv_heads; a.dim = B.dim; a.vdim = B.vdim; a.row = B.row; a.ring = B.ring; a.eps = e->cfg.rms_norm_eps; a.out = out; a.err_flag = e->ctx->d_err;
    uint32_t n = 0;
    const cudaError_t err = launch_window_attention(e->ctx->stream, b.f32, a, T, e->ctx->sm_count, &n, e->pdl);
    return engine_count(e, err, "attention", n);
}

bool mix_delta(KronosCudaEngine *e, Block &B, uint32_t T, const Act &out) {
    BlockModel &b = *e->blocks;
    cudaStream_t s = e->ctx->stream;
    DeltaArgs a{};
    a.in = b.z; a.in_stride = b.zs; a.decay = dense_view(B.decay->dm);
    a.decay_bias = B.decay_bias; a.rate_bias = B.rate_bias; a.norm = B.out_norm; a.state = B.state;
    a.decay_logit = b.logit; a.logit_stride = b.ls; a.rec = b.rec; a.o = b.scan_o;
    a.heads = B.heads; a.dim = B.dim; a.drow = B.row; a.rank = B.rank;
    a.decay_scale = B.decay_scale; a.unit_eps = B.unit_eps; a.eps = e->cfg.rms_norm_eps; a.out = out; a.err_flag = e->ctx->d_err;
    if (T == 1 && delta_step_fits(a)) return engine_count(e, launch_delta_step(s, b.f32, a, e->pdl), "recurrence");
    const Act r = act_of(b, b.act_s, T, B.rank);
    return engine_count(e, launch_delta_tanh(s, b.f32, a, r, T, e->pdl), "decay tanh") && product(e, B.decay, r, T, b.logit, b.ls, "decay product") &&
           engine_count(e, launch_delta_prompt(s, b.f32, a, T, e->ctx->sm_count, e->pdl), "recurrence", 3);
}

// The prompt path expands every cached position once per batch, the other works in latent space, where a pair of positions costs
// more (and runs on a slower kernel): the batch length from which the expansion pays.
bool latent_expands(const BlockModel &b, const Block &B, uint32_t T) {
    if (b.f32 || !B.flash || T < DENSE_TC_MIN) return false;
    const LatentShape &d = B.lat;
    const uint64_t direct = 2ull * (2 * d.kv_rank + d.rot_dim), expanded = d.dim + d.rot_dim + d.vdim, once = (uint64_t)d.kv_rank * (d.dim + d.vdim);
    return direct > expanded && (direct - expanded) * T > once;
}

bool mix_latent(KronosCudaEngine *e, Block &B, uint32_t T, const Act &out) {
    BlockModel &b = *e->blocks;
    cudaStream_t s = e->ctx->stream;
    const LatentShape &d = B.lat;
    LatentAttnArgs a{};
    a.d = d;
    a.in = a.q = b.z; a.in_stride = a.q_stride = b.zs;          // the query product takes the place of the latents once they are normed
    a.q_norm = B.q_latent_norm; a.kv_norm = B.kv_latent_norm; a.rot = B.rot; a.kv_up = dense_view(B.kv_up->dm);
    a.cache = Act{B.k, b.f32 ? d.row : B.ring.ring_len};
    a.pos = e->d_pos; a.scale = B.score_scale; a.eps = e->cfg.rms_norm_eps;
    a.q_lat = act_of(b, b.act_s, T, d.q_rank);
    a.part_o = b.part_o; a.part_m = b.part_m; a.part_l = b.part_l; a.out = out; a.err_flag = e->ctx->d_err;
    if (!engine_count(e, launch_latent_prep(s, b.f32, a, T, e->pdl), "latent norms") || !product(e, B.q_up, a.q_lat, T, b.z, b.zs, "query product")) return false;
    if (e->ctx_bound > 0 && latent_expands(b, B, T)) {
        a.q_rows = act_of(b, b.act_q, T, 0);
        a.kv = Act{b.act_kv, act_tokens(e->ctx_bound)};
        return product_act(e, B.kv_up, a.cache, e->ctx_bound, Epi::Panels, a.kv, "keys and values") &&
               engine_count(e, launch_latent_prompt(s, a, T, e->pdl), "attention", 2);
    }
    for (uint32_t t0 = 0; t0 < T; t0 += LATENT_TOKENS) {
        const uint32_t n = std::min(LATENT_TOKENS, T - t0);
        a.q_rows = act_of(b, b.act_q, n * d.heads, d.row);
        const uint32_t splits = latent_splits(d, n, e->ctx_bound > 0 ? e->ctx_bound : e->cfg.max_seq_len, e->ctx->sm_count);
        if (!engine_count(e, launch_latent_few(s, b.f32, a, t0, n, splits, e->pdl), "attention", 3)) return false;
    }
    return true;
}

NormArgs norm_args(const KronosCudaEngine *e, const float *post, const float *pre, const Act &out) {
    const BlockModel &b = *e->blocks;
    NormArgs a{};
    a.x = b.x; a.x_stride = b.hs; a.y = post ? b.proj : nullptr; a.y_stride = b.hs; a.post = post; a.pre = pre;
    a.mult = b.residual_mult; a.eps = e->cfg.rms_norm_eps; a.n = e->cfg.hidden_size; a.out = out;
    return a;
}
// residual of a sublayer (output in proj, norm weight `post`), norm in front of the next one
bool norm_add(KronosCudaEngine *e, const float *post, const float *pre, const Act &out, uint32_t T) {
    return engine_count(e, launch_block_norm(e->ctx->stream, e->blocks->f32, norm_args(e, post, pre, out), T, e->pdl), "residual norm");
}

// router, experts and shared expert on the normed activation ax, residual with norm `post`, norm `pre` in front of what follows
bool feed_experts(KronosCudaEngine *e, Block &B, const Act &ax, uint32_t T, const float *post, const float *pre) {
    BlockModel &b = *e->blocks;
    cudaStream_t s = e->ctx->stream;
    const uint32_t h = e->cfg.hidden_size, rows = up_rows(B.act, B.ff);
    RouteArgs r{};
    r.z = b.z; r.z_stride = b.zs; r.experts = B.experts; r.top = B.top; r.ids = b.route_ids; r.row = b.route_row; r.weight = b.route_w;
    r.act = epi_of(B.act); r.shared_ff = B.shared_ff; r.shared = act_of(b, b.act_s, T, B.shared_ff);
    const DenseView up = dense_view(B.expert_up[0]->dm), down = dense_view(B.expert_down[0]->dm);
    const ExpertView eu{B.d_up, rows, h, up.rows_pad, up.panels}, ed{B.d_down, h, B.ff, down.rows_pad, down.panels};
    if (!product(e, B.router, ax, T, b.z, b.zs, "router") || !engine_count(e, launch_route(s, b.f32, r, T, e->pdl), "expert choice")) return false;
    if (b.f32 || T < DENSE_TC_MIN) {
        const Act ae = act_of(b, b.act_e, T * B.top, B.ff);
        return engine_count(e, launch_expert_up(s, b.f32, r, eu, ax, ae, T, e->ctx->sm_count, e->pdl), "experts up") &&
               engine_count(e, launch_expert_down(s, b.f32, r, ed, ae, B.shared_down ? dense_view(B.shared_down->dm) : DenseView{}, b.proj, b.hs, T, e->ctx->sm_count, e->pdl), "experts down") &&
               norm_add(e, post, pre, ax, T);
    }
    const uint32_t packed = expert_rows(T, B.top, B.experts), items = expert_items(T, B.top, B.experts), tile = expert_tile(T, B.top, B.experts);
    const Act ap = act_of(b, b.act_p, packed, h), ae = act_of(b, b.act_e, packed, B.ff);
    NormArgs n = norm_args(e, post, pre, ax);
    n.top = B.top; n.pairs = b.pairs; n.pair_stride = b.hs; n.row = b.route_row; n.weight = b.route_w;
    return engine_count(e, launch_expert_plan(s, r, T, b.items, b.n_items, e->pdl), "expert plan") &&
           engine_count(e, launch_expert_gather(s, r, ax, h, ap, T, e->pdl), "expert gather") &&
           engine_count(e, launch_dense_experts(s, eu, ap, b.items, b.n_items, items, tile, DenseOut{r.act, nullptr, 0, 0.0f, ae}, e->ctx->d_err, e->pdl), "experts up") &&
           engine_count(e, launch_dense_experts(s, ed, ae, b.items, b.n_items, items, tile, dense_rows(b.pairs, b.hs), e->ctx->d_err, e->pdl), "experts down") &&
           (B.shared_down ? product(e, B.shared_down, r.shared, T, b.proj, b.hs, "shared expert down")
                          : cuda_ok(e->ctx, cudaMemsetAsync(b.proj, 0, (size_t)T * b.hs * 4, s), "clear")) &&
           engine_count(e, launch_block_norm(s, false, n, T, e->pdl), "residual norm");
}

// residual of the block's last sublayer (output in proj, norm weight w), then the token input, or the norm in front of the next block
bool finish_block(KronosCudaEngine *e, size_t l, const float *w, const float *pre, const Act &ax, uint32_t T) {
    BlockModel &b = *e->blocks;
    if (b.side_dim == 0) return norm_add(e, w, pre, ax, T);
    cudaStream_t s = e->ctx->stream;
    const Block &B = b.blocks[l];
    const SideArgs sd = side_args(e, l);
    const uint32_t h = e->cfg.hidden_size;
    if (T <= 16 && norm_side_fits(h, b.side_dim))
        return engine_count(e, launch_norm_side(s, b.f32, b.x, b.hs, b.proj, b.hs, w, h, e->cfg.rms_norm_eps, sd, ax, T, e->ctx->d_err, e->pdl), "residual norm + token input");
    const Act as = act_of(b, b.act_s, T, b.side_dim);
    return norm_add(e, w, nullptr, ax, T) && product(e, B.side_gate, ax, T, b.z, b.zs, "token input gate") &&
           engine_count(e, launch_side_gelu(s, b.f32, b.z, b.zs, sd, as, T, e->pdl), "token input gelu") &&
           product(e, B.side_proj, as, T, b.proj, b.hs, "token input proj") && norm_add(e, B.side_norm, nullptr, ax, T);
}

}  // namespace

bool blocks_enqueue(KronosCudaEngine *e, uint32_t T, bool embed, Tail tail) {
    BlockModel &b = *e->blocks;
    cudaStream_t s = e->ctx->stream;
    const uint32_t h = e->cfg.hidden_size, vocab = e->cfg.vocab_size;
    const uint64_t launches_before = e->ctx->launches;
    const Act ax = act_of(b, b.act_x, T, h);
    if (!embed) return fail(e->ctx, "block models run on token ids");
    if (!engine_count(e, launch_block_embed(s, b.f32, b.embed, e->d_token, h, b.x, b.hs, ax, T, false), "embed")) return false;
    if (b.blocks[0].pre1 && !norm_add(e, nullptr, b.blocks[0].pre1, ax, T)) return false;
    const bool fold_final = b.side_dim == 0 && (tail == Tail::AllLogits || (tail != Tail::None && T == 1));      // the last residual norm makes the head's activation
    for (size_t l = 0; l < b.blocks.size(); ++l) {
        Block &B = b.blocks[l];
        const Act am = act_of(b, b.act_m, T, B.o->dm.geom.cols);
        if (!product(e, B.in, ax, T, b.z, b.zs, "in-projection") ||
            !(B.mixer == KRONOS_CUDA_MIXER_WINDOW_ATTENTION ? mix_attention(e, B, T, am) : B.mixer == KRONOS_CUDA_MIXER_GENERAL_DELTA ? mix_delta(e, B, T, am) : mix_latent(e, B, T, am)) ||
            !product(e, B.o, am, T, b.proj, b.hs, "out-projection"))
            return false;
        const float *w = B.norm1, *next = l + 1 < b.blocks.size() ? b.blocks[l + 1].pre1 : fold_final ? b.final_norm : nullptr;
        if (B.ff > 0) {
            if (!norm_add(e, B.norm1, B.pre2, ax, T)) return false;
            if (B.experts > 0) {
                if (!feed_experts(e, B, ax, T, B.norm2, next)) return false;
                continue;
            }
            const Act af = act_of(b, b.act_m, T, B.ff);
            const bool up = B.act == KRONOS_CUDA_ACT_POLYNORM
                                ? product(e, B.up, ax, T, b.z, b.zs, "up") && engine_count(e, launch_polynorm(s, b.f32, b.z, b.zs, B.ff, B.coef, e->cfg.rms_norm_eps, af, T, e->pdl), "activation")
                                : product_act(e, B.up, ax, T, epi_of(B.act), af, "up");
            if (!up || !product(e, B.down, af, T, b.proj, b.hs, "down")) return false;
            w = B.norm2;
        }
        if (!finish_block(e, l, w, next, ax, T)) return false;
    }
    if (tail != Tail::None) {
        const uint32_t t0 = tail == Tail::AllLogits ? 0 : T - 1, n = T - t0;
        Act af = ax;
        if (!fold_final) {
            af = act_of(b, b.act_m, n, h);
            NormArgs a = norm_args(e, nullptr, b.final_norm, af);
            a.x += (size_t)t0 * b.hs;
            if (!engine_count(e, launch_block_norm(s, b.f32, a, n, e->pdl), "final norm")) return false;
        }
        if (!product_out(e, b.head, af, n, DenseOut{b.softcap > 0.0f ? Epi::Softcap : Epi::Rows, e->logits, vocab, b.softcap, Act{}}, "head")) return false;
    }
    const bool ok = tail == Tail::Greedy
                        ? engine_count(e, launch_argmax_step(s, e->logits, vocab, e->d_token, e->d_pos, e->d_history, e->d_step, e->argmax_scratch, e->pdl), "argmax")
                        : engine_count(e, launch_advance_pos(s, e->d_pos, T, e->pdl), "advance");
    if (T == 1) b.step_launches = (uint32_t)(e->ctx->launches - launches_before);
    return ok;
}

uint32_t blocks_step_launches(const KronosCudaEngine *e) { return e->blocks->step_launches; }
const float *blocks_hidden(const KronosCudaEngine *e) { return e->blocks->x + (size_t)e->last_row * e->blocks->hs; }

bool blocks_can_continue(const KronosCudaEngine *e, size_t pos) {
    const BlockModel &b = *e->blocks;
    if (pos == 0) return true;
    if (b.pos == LOST) return false;
    // without recurrent state an earlier position is as good, while the rings still hold the rows it sees
    return pos == b.pos || (!b.recurrent && pos < b.pos && (!b.windowed || b.pos - pos <= e->max_batch));
}

bool blocks_begin(KronosCudaEngine *e, bool token_ids, size_t pos) {
    BlockModel &b = *e->blocks;
    if (!token_ids) return fail(e->ctx, "forward: block models run on token ids");
    if (!blocks_can_continue(e, pos))
        return fail(e->ctx, "forward: the sequence stands at position " + (b.pos == LOST ? std::string("(lost)") : std::to_string(b.pos)) +
                                ": continue there, restore a snapshot, or start again at 0");
    if (pos == 0)
        for (Block &B : b.blocks)
            if (B.state && !cuda_ok(e->ctx, cudaMemsetAsync(B.state, 0, B.state_floats * 4, e->ctx->stream), "clear state")) return false;
    b.pos = LOST;
    return true;
}
void blocks_end(KronosCudaEngine *e, size_t pos) { e->blocks->pos = pos; }

bool blocks_park_state(KronosCudaEngine *e, bool save) {
    BlockModel &b = *e->blocks;
    size_t i = 0;
    for (Block &B : b.blocks) {
        if (!B.state) continue;
        if (b.parked.size() <= i) {
            float *p = nullptr;
            if (!dev_alloc(e, p, B.state_floats)) return false;
            b.parked.push_back(p);
        }
        if (!cuda_ok(e->ctx, cudaMemcpyAsync(save ? b.parked[i] : B.state, save ? B.state : b.parked[i], B.state_floats * 4, cudaMemcpyDeviceToDevice, e->ctx->stream), "park state")) return false;
        ++i;
    }
    return true;
}

size_t blocks_kv_bytes(const KronosCudaEngine *e, size_t positions) {
    size_t n = 0;
    for (const Block &B : e->blocks->blocks)
        if (B.k) n += std::min<size_t>(positions, B.ring.window ? B.ring.window : B.ring.ring_len) * (B.v ? B.kv_heads * (B.dim + B.vdim) : B.lat.kv_rank + B.lat.rot_dim) * (e->blocks->f32 ? 4 : 2);
    return n;
}

// Snapshot of the sequence: header {"K2TBLOCK", position, bytes of the rest}, then per block its key and value rings, latent rows or state.
static const char SNAPSHOT_MAGIC[8] = {'K', '2', 'T', 'B', 'L', 'O', 'C', 'K'};
size_t blocks_snapshot_bytes(const KronosCudaEngine *e) {
    size_t n = 24;
    for (const Block &B : e->blocks->blocks) n += B.k_bytes + B.v_bytes + B.state_floats * 4;
    return n;
}
bool blocks_save(KronosCudaEngine *e, size_t n, size_t cur_pos, uint8_t *out) {
    BlockModel &b = *e->blocks;
    if (cur_pos != b.pos || n < cur_pos) return fail(e->ctx, "save_kv_prefix: a recurrent state can only be saved where the sequence stands");
    const uint64_t head[2] = {b.pos, blocks_snapshot_bytes(e) - 24};
    std::memcpy(out, SNAPSHOT_MAGIC, 8);
    std::memcpy(out + 8, head, 16);
    out += 24;
    for (Block &B : b.blocks) {
        const struct { const void *p; size_t n; } parts[3] = {{B.k, B.k_bytes}, {B.v, B.v_bytes}, {B.state, B.state_floats * 4}};
        for (const auto &part : parts) {
            if (part.n && !cuda_ok(e->ctx, cudaMemcpyAsync(out, part.p, part.n, cudaMemcpyDeviceToHost, e->ctx->stream), "save_kv_prefix")) return false;
            out += part.n;
        }
    }
    return sync_and_check(e->ctx, "save_kv_prefix");
}
bool blocks_restore(KronosCudaEngine *e, const uint8_t *data, size_t len) {
    BlockModel &b = *e->blocks;
    uint64_t head[2];
    if (len != blocks_snapshot_bytes(e) || std::memcmp(data, SNAPSHOT_MAGIC, 8) != 0) return fail(e->ctx, "restore_kv_prefix: not a snapshot of this model");
    std::memcpy(head, data + 8, 16);
    if (head[1] != len - 24 || head[0] > e->cfg.max_seq_len) return fail(e->ctx, "restore_kv_prefix: not a snapshot of this model");
    b.pos = LOST;
    data += 24;
    for (Block &B : b.blocks) {
        const struct { void *p; size_t n; } parts[3] = {{B.k, B.k_bytes}, {B.v, B.v_bytes}, {B.state, B.state_floats * 4}};
        for (const auto &part : parts) {
            if (part.n && !cuda_ok(e->ctx, cudaMemcpyAsync(part.p, data, part.n, cudaMemcpyHostToDevice, e->ctx->stream), "restore_kv_prefix")) return false;
            data += part.n;
        }
    }
    if (!sync_and_check(e->ctx, "restore_kv_prefix")) return false;
    b.pos = head[0];
    return true;
}

void blocks_destroy(KronosCudaEngine *e) {
    if (!e->blocks) return;
    for (Block &B : e->blocks->blocks) {
        for (KronosCudaMatrix *m : {B.in, B.decay, B.o, B.up, B.down, B.side_gate, B.side_proj, B.q_up, B.kv_up, B.router, B.shared_down})
            if (m) kronos_cuda_matrix_free(e->ctx, m);
        for (auto *list : {&B.expert_up, &B.expert_down})
            for (KronosCudaMatrix *m : *list)
                if (m) kronos_cuda_matrix_free(e->ctx, m);
    }
    if (e->blocks->head) kronos_cuda_matrix_free(e->ctx, e->blocks->head);
    delete e->blocks;
    e->blocks = nullptr;
}

}  // namespace k2t

using namespace k2t;

extern "C" KronosCudaEngine *kronos_cuda_engine_create_blocks(KronosCudaContext *ctx, const KronosCudaBlocksConfig *cfg, const KronosCudaBlockDesc *descs, size_t n_blocks,
                                                              const float *final_norm, const KronosCudaMatrixDesc *head, const uint16_t *embed_bf16,
                                                              const uint16_t *side_embed_bf16) {
    if (!ctx) return nullptr;
    ctx->err.clear();
    auto refuse = [&](const std::string &why) { fail(ctx, "engine_create_blocks: " + why); return (KronosCudaEngine *)nullptr; };
    if (!cfg || !descs || !final_norm || !head || !embed_bf16) return refuse("NULL argument");
    const KronosCudaBlocksConfig &c = *cfg;
    if (c.struct_size != sizeof(KronosCudaBlocksConfig)) return refuse("config.struct_size does not match this library (binding out of date?)");
    if (n_blocks == 0 || n_blocks != c.num_blocks) return refuse("n_blocks does not match the config");
    if (c.hidden_size == 0 || c.vocab_size == 0 || c.max_seq_len == 0) return refuse("a size is 0");
    if (c.precision != 16 && c.precision != 32) return refuse("precision must be 16 or 32");
    if (!(c.residual_mult > 0.0f) || !(c.logit_softcap >= 0.0f)) return refuse("residual_mult must be positive, logit_softcap not negative");
    if (c.side_dim > 0 && c.residual_mult != 1.0f) return refuse("the token input goes with residual_mult 1");
    if ((c.side_dim > 0) != (side_embed_bf16 != nullptr)) return refuse("side_dim and the side embedding table go together");
    if (!make_current(ctx)) return nullptr;
    KronosCudaEngine *e = new (std::nothrow) KronosCudaEngine();
    BlockModel *b = new (std::nothrow) BlockModel();
    if (!e || !b) { delete e; delete b; return refuse("out of host memory"); }
    e->ctx = ctx;
    e->blocks = b;
    e->cfg.hidden_size = c.hidden_size; e->cfg.num_layers = c.num_blocks; e->cfg.vocab_size = c.vocab_size; e->cfg.max_seq_len = c.max_seq_len;
    e->cfg.rms_norm_eps = c.rms_norm_eps;
    e->layers.resize(n_blocks);
    e->max_batch = 2048;                       // tokens per prompt batch: the row tiles of a projection times 256-token tiles fill the SMs
    if (const char *v = std::getenv("KRONOS_CUDA_PROMPT_BATCH")) e->max_batch = std::min(4096u, std::max(16u, ((uint32_t)std::strtoul(v, nullptr, 10) + 15u) & ~15u));
    e->max_batch = std::min(e->max_batch, std::max(16u, (c.max_seq_len + 15u) & ~15u));
    if (const char *v = std::getenv("KRONOS_CUDA_PDL")) e->pdl = v[0] != '0';
    b->f32 = c.precision == 32;
    b->side_dim = c.side_dim;
    b->residual_mult = c.residual_mult;
    b->softcap = c.logit_softcap;
    b->hs = pad8(c.hidden_size);
    b->blocks.resize(n_blocks);
    const uint32_t h = c.hidden_size, MB = e->max_batch, bits = c.precision;
    auto bad = [&](const std::string &why) { const std::string keep = why; kronos_cuda_engine_destroy(e); return refuse(keep); };
    auto upload = [&](KronosCudaMatrix *&m, const KronosCudaMatrixDesc &d, uint32_t rows, uint32_t cols) {
        if (d.kind != KRONOS_CUDA_MATRIX_DENSE || d.bits != bits || d.rows != rows || d.cols != cols) { fail(ctx, "a matrix is not dense in the engine's precision or has the wrong shape"); return false; }
        m = kronos_cuda_matrix_upload(ctx, &d, 0);
        if (m) e->weight_bytes += m->dm.geom.file_bytes;
        return m != nullptr;
    };
    auto vec = [&](float *&p, const float *src, uint32_t n) {      // read four at a time: padded with zeros
        if (!src) { fail(ctx, "a vector is missing"); return false; }
        return dev_alloc(e, p, pad8(n)) && cuda_ok(ctx, cudaMemcpyAsync(p, src, (size_t)n * 4, cudaMemcpyHostToDevice, ctx->stream), "upload");
    };
    // a matrix cut into parts of equal shape, one below the other
    auto part = [&](const KronosCudaMatrixDesc &d, uint32_t i, uint32_t rows) {
        KronosCudaMatrixDesc p = d;
        p.rows = rows;
        p.len0 = (size_t)rows * d.cols * (bits / 8);
        p.data0 = d.data0 + i * p.len0;
        return p;
    };
    auto whole = [&](const KronosCudaMatrixDesc &d, uint64_t rows, uint32_t cols) {
        return d.kind == KRONOS_CUDA_MATRIX_DENSE && d.bits == bits && d.rows == rows && d.cols == cols && d.data0 && d.len0 >= rows * cols * (bits / 8);
    };
    auto upload_parts = [&](std::vector<KronosCudaMatrix *> &list, const void **&table, const KronosCudaMatrixDesc &d, uint32_t n, uint32_t rows, uint32_t cols) {
        if (!whole(d, (uint64_t)n * rows, cols)) { fail(ctx, "the experts' matrices are not dense in the engine's precision or have the wrong shape"); return false; }
        list.resize(n);
        std::vector<const void *> base(n);
        for (uint32_t i = 0; i < n; ++i) {
            if (!upload(list[i], part(d, i, rows), rows, cols)) return false;
            base[i] = list[i]->dm.d_base;
        }
        return dev_alloc(e, table, n, base.data()) && cuda_ok(ctx, cudaStreamSynchronize(ctx->stream), "upload");
    };
    std::map<const float *, float *> rot_tables;
    uint32_t z_cols = std::max(8u, c.side_dim), m_cols = h, s_cols = std::max(1u, c.side_dim), logit_cols = 0;
    size_t q_elems = 0, rec_floats = 0, o_floats = 0, qa_bytes = 0, kv_bytes = 0, part_floats = 0, part_rows = 0;
    uint32_t routes = 0, packed_max = 0, items_max = 0, expert_ff = 0;
    for (size_t l = 0; l < n_blocks; ++l) {
        const KronosCudaBlockDesc &d = descs[l];
        Block &B = b->blocks[l];
        const std::string at = "block " + std::to_string(l) + ": ";
        B.mixer = d.mixer; B.heads = d.heads; B.kv_heads = d.kv_heads; B.dim = d.dim; B.vdim = d.vdim; B.ff = d.ff;
        if (B.heads == 0 || B.dim == 0) return bad(at + "no heads");
        B.act = d.act; B.experts = d.experts; B.top = d.experts_top; B.shared_ff = d.shared_ff;
        if (!vec(B.norm1, d.norm1, h) || (d.pre_norm1 && !vec(B.pre1, d.pre_norm1, h)) || (d.pre_norm2 && !vec(B.pre2, d.pre_norm2, h))) return bad(at + ctx->err);
        if (c.side_dim > 0 && (B.pre1 || B.pre2 || B.experts)) return bad(at + "the token input does not go with norms in front of the sublayers or with experts");
        uint32_t mix_cols = 0;
        if (d.mixer == KRONOS_CUDA_MIXER_WINDOW_ATTENTION) {
            if (B.kv_heads == 0 || B.heads % B.kv_heads || B.vdim == 0) return bad(at + "query heads must be a multiple of the key/value heads");
            B.row = window_attn_row(B.dim, B.vdim);
            if (B.row == 0) return bad(at + "attention: head sizes up to 256");
            if (!window_attn_fits(b->f32, B.heads / B.kv_heads, B.row)) return bad(at + "attention: too many query heads per key/value head for this head size");
            const uint32_t rows = B.heads * B.dim + B.kv_heads * (B.dim + B.vdim);
            mix_cols = B.heads * B.vdim;
            if (!vec(B.q_norm, d.q_norm, B.dim) || !vec(B.k_norm, d.k_norm, B.dim) || !vec(B.head_scale, d.head_scale, B.heads) || !vec(B.head_slope, d.head_slope, B.heads) ||
                !upload(B.in, d.in_proj, rows, h))
                return bad(at + ctx->err);
            // a prompt batch stores its rows before any of its tokens attends, so the ring holds a window and a batch
            const uint64_t need = d.window == 0 ? c.max_seq_len : std::min<uint64_t>(c.max_seq_len, (uint64_t)d.window + MB);
            B.ring.window = d.window; B.ring.sinks = 0; B.ring.ring_len = (uint32_t)((need + 63) & ~63ull);
            B.k_bytes = B.v_bytes = (size_t)B.kv_heads * B.ring.ring_len * B.row * (bits / 8);
            b->windowed = b->windowed || d.window > 0;
            e->kv_rows = std::max(e->kv_rows, B.ring.ring_len);
            if (!dev_alloc(e, B.k, B.k_bytes) || !dev_alloc(e, B.v, B.v_bytes)) return bad(at + ctx->err);
            z_cols = std::max(z_cols, rows);
            q_elems = std::max(q_elems, (size_t)B.heads * B.row);
        } else if (d.mixer == KRONOS_CUDA_MIXER_GENERAL_DELTA) {
            B.rank = d.decay_rank; B.decay_scale = d.decay_scale; B.unit_eps = d.unit_eps;
            B.row = delta_row(B.dim);
            if (B.row == 0 || B.rank == 0) return bad(at + "delta rule: head sizes up to 256, decay rank at least 1");
            const uint32_t hd = B.heads * B.dim, rows = 5 * hd + B.rank;
            mix_cols = hd;
            if (!vec(B.decay_bias, d.decay_bias, hd) || !vec(B.rate_bias, d.rate_bias, hd) || !vec(B.out_norm, d.out_norm, hd) || !upload(B.in, d.in_proj, rows, h) ||
                !upload(B.decay, d.decay_proj, hd, B.rank))
                return bad(at + ctx->err);
            B.state_floats = (size_t)B.heads * B.row * B.row;
            if (!dev_alloc(e, B.state, B.state_floats)) return bad(at + ctx->err);
            b->recurrent = true;
            z_cols = std::max(z_cols, rows);
            s_cols = std::max(s_cols, B.rank);
            logit_cols = std::max(logit_cols, hd);
            rec_floats = std::max(rec_floats, delta_record_floats(MB, B.heads, B.row));
            o_floats = std::max(o_floats, (size_t)B.heads * B.row);
        } else if (d.mixer == KRONOS_CUDA_MIXER_LATENT_ATTENTION) {
            if (B.vdim == 0 || d.q_rank == 0 || d.kv_rank == 0 || d.rot_dim == 0 || d.rot_dim % 2) return bad(at + "latent attention: a size is 0, or rot_dim is odd");
            if (!(d.score_scale > 0.0f) || !d.rot_cos_sin) return bad(at + "latent attention: score_scale must be positive, and the rotation table is needed");
            const LatentShape lat = latent_shape(b->f32, B.heads, B.dim, d.rot_dim, B.vdim, d.q_rank, d.kv_rank);
            B.lat = lat;
            B.score_scale = d.score_scale;
            if (!latent_attn_fits(b->f32, lat)) return bad(at + "latent attention: kv_rank up to 1024, and rows that fit in shared memory");
            B.flash = !b->f32 && latent_flash_fits(lat);
            const uint32_t rows = d.q_rank + d.kv_rank + d.rot_dim, q_rows = B.heads * (B.dim + d.rot_dim), dc = latent_head_cols(B.dim), vc = latent_head_cols(B.vdim);
            mix_cols = B.heads * B.vdim;
            if (!whole(d.kv_up, (uint64_t)B.heads * (B.dim + B.vdim), d.kv_rank)) return bad(at + "kv_up is not dense in the engine's precision or has the wrong shape");
            // every head starts a panel of the expanded keys and values: its rows are padded with zeros
            std::vector<uint8_t> padded((size_t)B.heads * (dc + vc) * d.kv_rank * (bits / 8), 0);
            const size_t row_bytes = (size_t)d.kv_rank * (bits / 8);
            for (uint32_t i = 0; i < B.heads; ++i) {
                std::memcpy(padded.data() + (size_t)i * dc * row_bytes, d.kv_up.data0 + (size_t)i * B.dim * row_bytes, B.dim * row_bytes);
                std::memcpy(padded.data() + ((size_t)B.heads * dc + (size_t)i * vc) * row_bytes, d.kv_up.data0 + ((size_t)B.heads * B.dim + (size_t)i * B.vdim) * row_bytes, B.vdim * row_bytes);
            }
            KronosCudaMatrixDesc kv = d.kv_up;
            kv.rows = B.heads * (dc + vc); kv.data0 = padded.data(); kv.len0 = padded.size();
            float *&rot = rot_tables[d.rot_cos_sin];
            if (!rot && !dev_alloc(e, rot, (size_t)c.max_seq_len * d.rot_dim, d.rot_cos_sin)) return bad(at + ctx->err);
            B.rot = rot;
            if (!vec(B.q_latent_norm, d.q_latent_norm, d.q_rank) || !vec(B.kv_latent_norm, d.kv_latent_norm, d.kv_rank) || !upload(B.in, d.in_proj, rows, h) ||
                !upload(B.q_up, d.q_up, q_rows, d.q_rank) || !upload(B.kv_up, kv, kv.rows, d.kv_rank) || !cuda_ok(ctx, cudaStreamSynchronize(ctx->stream), "upload"))
                return bad(at + ctx->err);
            B.ring.window = B.ring.sinks = 0;
            B.ring.ring_len = (c.max_seq_len + 127) & ~127u;
            e->kv_rows = std::max(e->kv_rows, B.ring.ring_len);
            B.k_bytes = (size_t)B.ring.ring_len * lat.row * (bits / 8);
            if (!dev_alloc(e, B.k, B.k_bytes + (size_t)DENSE_TOK_SLACK * PANEL * 2)) return bad(at + ctx->err);          // a token tile of the expanding product may read beyond
            z_cols = std::max({z_cols, rows, q_rows});
            s_cols = std::max(s_cols, d.q_rank);
            qa_bytes = std::max(qa_bytes, act_bytes(b->f32, std::min(LATENT_TOKENS, MB) * B.heads, lat.row));
            part_rows = std::max(part_rows, std::max((size_t)32 * ctx->sm_count, (size_t)LATENT_TOKENS * B.heads));
            part_floats = std::max(part_floats, part_rows * ((d.kv_rank + 3u) & ~3u));
            if (B.flash) {
                qa_bytes = std::max(qa_bytes, act_bytes(false, MB, B.heads * (dc + latent_head_cols(d.rot_dim))));
                kv_bytes = std::max(kv_bytes, act_bytes(false, B.ring.ring_len, kv.rows));
            }
        } else {
            return bad(at + "unknown mixer " + std::to_string(d.mixer));
        }
        if (!upload(B.o, d.o_proj, h, mix_cols)) return bad(at + ctx->err);
        m_cols = std::max(m_cols, mix_cols);
        if (B.ff > 0) {
            const uint32_t rows = up_rows(B.act, B.ff), shared_rows = up_rows(B.act, B.shared_ff);
            if (B.act > KRONOS_CUDA_ACT_RELU_SQUARED) return bad(at + "unknown activation " + std::to_string(B.act));
            if (!vec(B.norm2, d.norm2, h)) return bad(at + ctx->err);
            if (B.experts == 0) {
                if ((B.act == KRONOS_CUDA_ACT_POLYNORM && !vec(B.coef, d.act_coef, 4)) || !upload(B.up, d.up_proj, rows, h) || !upload(B.down, d.down_proj, h, B.ff)) return bad(at + ctx->err);
                z_cols = std::max(z_cols, rows);
                m_cols = std::max(m_cols, B.ff);
            } else {
                if (B.act == KRONOS_CUDA_ACT_POLYNORM) return bad(at + "experts take a gated gelu or a squared relu");
                if (B.experts > ROUTE_MAX_EXPERTS || B.top == 0 || B.top > B.experts || B.top > 32) return bad(at + "experts: at most 1024, of which a token takes 1 to 32");
                if (!upload(B.router, d.router, B.experts + shared_rows, h) || (B.shared_ff > 0 && !upload(B.shared_down, d.shared_down, h, B.shared_ff)) ||
                    !upload_parts(B.expert_up, B.d_up, d.up_proj, B.experts, rows, h) || !upload_parts(B.expert_down, B.d_down, d.down_proj, B.experts, h, B.ff))
                    return bad(at + ctx->err);
                z_cols = std::max(z_cols, B.experts + shared_rows);
                s_cols = std::max(s_cols, B.shared_ff);
                routes = std::max(routes, MB * B.top);
                packed_max = std::max(packed_max, expert_rows(MB, B.top, B.experts));
                items_max = std::max(items_max, MB * B.top / EXPERT_TILE_MIN + B.experts);
                expert_ff = std::max(expert_ff, B.ff);
            }
        }
        if (c.side_dim > 0 && (!vec(B.side_norm, d.side_norm, h) || !upload(B.side_gate, d.side_gate, c.side_dim, h) || !upload(B.side_proj, d.side_proj, h, c.side_dim)))
            return bad(at + ctx->err);
    }
    b->zs = pad8(z_cols);
    b->ls = pad8(logit_cols);
    auto act = [&](void *&p, uint32_t cols) { uint8_t *q = nullptr; const bool ok = dev_alloc(e, q, act_bytes(b->f32, MB, cols)); p = q; return ok; };
    uint8_t *q = nullptr, *qa = nullptr, *kva = nullptr, *pa = nullptr, *ea = nullptr;
    if (!upload(b->head, *head, c.vocab_size, h) || !vec(b->final_norm, final_norm, h) || !dev_alloc(e, b->embed, (size_t)c.vocab_size * h, embed_bf16) ||
        (side_embed_bf16 && !dev_alloc(e, b->side_embed, (size_t)c.vocab_size * c.side_dim * n_blocks, side_embed_bf16)) ||
        !dev_alloc(e, b->x, (size_t)MB * b->hs) || !dev_alloc(e, b->z, (size_t)MB * b->zs) || !dev_alloc(e, b->proj, (size_t)MB * b->hs) || !dev_alloc(e, b->logit, (size_t)MB * b->ls) ||
        !dev_alloc(e, b->rec, rec_floats) || !dev_alloc(e, b->scan_o, (size_t)MB * o_floats) || !act(b->act_x, h) || !act(b->act_m, m_cols) || !act(b->act_s, s_cols) ||
        (qa_bytes && !(dev_alloc(e, qa, qa_bytes) && dev_alloc(e, kva, kv_bytes) && dev_alloc(e, b->part_o, part_floats) && dev_alloc(e, b->part_m, part_rows) && dev_alloc(e, b->part_l, part_rows))) ||
        (routes && !(dev_alloc(e, b->route_ids, routes) && dev_alloc(e, b->route_row, routes) && dev_alloc(e, b->route_w, routes) && dev_alloc(e, b->n_items, 1) && dev_alloc(e, b->items, items_max) &&
                     dev_alloc(e, pa, b->f32 ? 0 : act_bytes(false, packed_max, h)) && dev_alloc(e, ea, act_bytes(b->f32, packed_max, expert_ff)) &&
                     dev_alloc(e, b->pairs, b->f32 ? 0 : (size_t)packed_max * b->hs))) ||
        !dev_alloc(e, q, (size_t)MB * q_elems * (bits / 8)) || !dev_alloc(e, e->logits, (size_t)MB * c.vocab_size) || !dev_alloc(e, e->d_token, MB) || !dev_alloc(e, e->d_pos, 1) ||
        !dev_alloc(e, e->d_step, 1) || !dev_alloc(e, e->d_history, c.max_seq_len) || !dev_alloc(e, e->d_dbg, 32) || !dev_alloc(e, e->argmax_scratch, ARGMAX_SCRATCH_WORDS) ||
        !cuda_ok(ctx, cudaStreamSynchronize(ctx->stream), "engine_create_blocks"))
        return bad(ctx->err);
    b->q = q;
    b->act_q = qa; b->act_kv = kva; b->act_p = pa; b->act_e = ea;
    e->mega_why = "block models are served by the per-operator path";
    return e;
}
