// Models described block by block: every block names its token mixer (sliding-window attention or the generalized delta rule),
// its feed-forward (or none) and its sizes, over unquantized matrices.  Post-normed residual: x += norm1(mixer(x)),
// x += norm2(ff(x)), then the optional per-layer token input.  The engine around it - graphs, prompt batches, greedy loop, argmax,
// launch counting, profiling - is k2t_engine.cu's; here are creation, the state manager (a key/value ring per attention layer, a
// state matrix per head of a recurrent layer, the sequence's position) and the launches of a batch.
//
// One decoded token: attention block = in-projection, attention (norms, cache row, softmax, one cluster launch), out-projection,
// residual norm, up, activation, down, residual norm + token input (one cluster launch); recurrent block without feed-forward =
// in-projection, recurrence (one launch), out-projection, residual norm + token input.
#include <cmath>
#include <cstdlib>
#include <cstring>
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
    // attention: ring of key and value rows; recurrent: state [heads][row][row]
    KvRing ring{};
    uint8_t *k = nullptr, *v = nullptr;
    size_t cache_bytes = 0;                    // of k, and of v
    float *state = nullptr;
    size_t state_floats = 0;
};

struct BlockModel {
    bool f32 = false, recurrent = false;
    uint32_t side_dim = 0, hs = 0;             // hs: stride of fp32 hidden-sized rows
    std::vector<Block> blocks;
    KronosCudaMatrix *head = nullptr;
    float *final_norm = nullptr;
    uint16_t *embed = nullptr, *side_embed = nullptr;
    // workspace, max_batch tokens
    float *x = nullptr, *z = nullptr, *proj = nullptr, *logit = nullptr, *rec = nullptr, *scan_o = nullptr;
    void *act_x = nullptr, *act_m = nullptr, *act_s = nullptr, *q = nullptr;
    size_t zs = 0, ls = 0;                     // strides of z and of the decay logits
    std::vector<float *> parked;               // copies of the recurrent states
    size_t pos = 0;                            // where the sequence stands
    uint32_t step_launches = 0;
};

namespace {

constexpr size_t LOST = ~(size_t)0;
constexpr uint32_t pad8(uint32_t n) { return (n + 7u) & ~7u; }

Act act_of(const BlockModel &b, void *p, uint32_t T, uint32_t cols) { return Act{p, act_ld(b.f32, T, cols)}; }

bool product(KronosCudaEngine *e, const KronosCudaMatrix *m, const Act &x, uint32_t T, float *out, size_t stride, const char *what) {
    uint32_t n = 0;
    const cudaError_t err = launch_dense(e->ctx->stream, m->dm, x, T, out, stride, e->ctx->sm_count, e->ctx->d_err, &n, e->pdl);
    return engine_count(e, err, what, n);
}

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

bool norm_add(KronosCudaEngine *e, const float *w, const Act &out, uint32_t T) {
    BlockModel &b = *e->blocks;
    return engine_count(e, launch_block_norm(e->ctx->stream, b.f32, true, b.x, b.hs, b.proj, b.hs, w, e->cfg.hidden_size, e->cfg.rms_norm_eps, out, T, e->pdl), "residual norm");
}

// residual of the block's last sublayer (output in proj, norm weight w), then the token input
bool finish_block(KronosCudaEngine *e, size_t l, const float *w, const Act &ax, uint32_t T) {
    BlockModel &b = *e->blocks;
    if (b.side_dim == 0) return norm_add(e, w, ax, T);
    cudaStream_t s = e->ctx->stream;
    const Block &B = b.blocks[l];
    const SideArgs sd = side_args(e, l);
    const uint32_t h = e->cfg.hidden_size;
    if (T <= 16 && norm_side_fits(h, b.side_dim))
        return engine_count(e, launch_norm_side(s, b.f32, b.x, b.hs, b.proj, b.hs, w, h, e->cfg.rms_norm_eps, sd, ax, T, e->ctx->d_err, e->pdl), "residual norm + token input");
    const Act as = act_of(b, b.act_s, T, b.side_dim);
    return norm_add(e, w, ax, T) && product(e, B.side_gate, ax, T, b.z, b.zs, "token input gate") &&
           engine_count(e, launch_side_gelu(s, b.f32, b.z, b.zs, sd, as, T, e->pdl), "token input gelu") &&
           product(e, B.side_proj, as, T, b.proj, b.hs, "token input proj") && norm_add(e, B.side_norm, ax, T);
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
    for (size_t l = 0; l < b.blocks.size(); ++l) {
        Block &B = b.blocks[l];
        const bool attn = B.mixer == KRONOS_CUDA_MIXER_WINDOW_ATTENTION;
        const Act am = act_of(b, b.act_m, T, B.o->dm.geom.cols);
        if (!product(e, B.in, ax, T, b.z, b.zs, "in-projection") || !(attn ? mix_attention(e, B, T, am) : mix_delta(e, B, T, am)) ||
            !product(e, B.o, am, T, b.proj, b.hs, "out-projection"))
            return false;
        const float *w = B.norm1;
        if (B.ff > 0) {
            const Act af = act_of(b, b.act_m, T, B.ff);
            if (!norm_add(e, B.norm1, ax, T) || !product(e, B.up, ax, T, b.z, b.zs, "up") ||
                !engine_count(e, launch_polynorm(s, b.f32, b.z, b.zs, B.ff, B.coef, e->cfg.rms_norm_eps, af, T, e->pdl), "activation") ||
                !product(e, B.down, af, T, b.proj, b.hs, "down"))
                return false;
            w = B.norm2;
        }
        if (!finish_block(e, l, w, ax, T)) return false;
    }
    if (tail != Tail::None) {
        const uint32_t t0 = tail == Tail::AllLogits ? 0 : T - 1, n = T - t0;
        const Act af = act_of(b, b.act_m, n, h);
        if (!engine_count(e, launch_block_norm(s, b.f32, false, b.x + (size_t)t0 * b.hs, b.hs, nullptr, 0, b.final_norm, h, e->cfg.rms_norm_eps, af, n, e->pdl), "final norm") ||
            !product(e, b.head, af, n, e->logits, vocab, "head"))
            return false;
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
    return pos == b.pos || (!b.recurrent && pos < b.pos && b.pos - pos <= e->max_batch);
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
        if (B.k) n += std::min<size_t>(positions, B.ring.window ? B.ring.window : B.ring.ring_len) * B.kv_heads * (B.dim + B.vdim) * (e->blocks->f32 ? 4 : 2);
    return n;
}

// Snapshot of the sequence: header {"K2TBLOCK", position, bytes of the rest}, then per block its key ring, value ring or state.
static const char SNAPSHOT_MAGIC[8] = {'K', '2', 'T', 'B', 'L', 'O', 'C', 'K'};
size_t blocks_snapshot_bytes(const KronosCudaEngine *e) {
    size_t n = 24;
    for (const Block &B : e->blocks->blocks) n += 2 * B.cache_bytes + B.state_floats * 4;
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
        const struct { const void *p; size_t n; } parts[3] = {{B.k, B.cache_bytes}, {B.v, B.cache_bytes}, {B.state, B.state_floats * 4}};
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
        const struct { void *p; size_t n; } parts[3] = {{B.k, B.cache_bytes}, {B.v, B.cache_bytes}, {B.state, B.state_floats * 4}};
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
    for (Block &B : e->blocks->blocks)
        for (KronosCudaMatrix *m : {B.in, B.decay, B.o, B.up, B.down, B.side_gate, B.side_proj})
            if (m) kronos_cuda_matrix_free(e->ctx, m);
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
    uint32_t z_cols = std::max(8u, c.side_dim), m_cols = h, s_cols = std::max(1u, c.side_dim), logit_cols = 0;
    size_t q_elems = 0, rec_floats = 0, o_floats = 0;
    for (size_t l = 0; l < n_blocks; ++l) {
        const KronosCudaBlockDesc &d = descs[l];
        Block &B = b->blocks[l];
        const std::string at = "block " + std::to_string(l) + ": ";
        B.mixer = d.mixer; B.heads = d.heads; B.kv_heads = d.kv_heads; B.dim = d.dim; B.vdim = d.vdim; B.ff = d.ff;
        if (B.heads == 0 || B.dim == 0) return bad(at + "no heads");
        if (!vec(B.norm1, d.norm1, h)) return bad(at + ctx->err);
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
            B.cache_bytes = (size_t)B.kv_heads * B.ring.ring_len * B.row * (bits / 8);
            e->kv_rows = std::max(e->kv_rows, B.ring.ring_len);
            if (!dev_alloc(e, B.k, B.cache_bytes) || !dev_alloc(e, B.v, B.cache_bytes)) return bad(at + ctx->err);
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
        } else {
            return bad(at + "unknown mixer " + std::to_string(d.mixer));
        }
        if (!upload(B.o, d.o_proj, h, mix_cols)) return bad(at + ctx->err);
        m_cols = std::max(m_cols, mix_cols);
        if (B.ff > 0) {
            if (!vec(B.norm2, d.norm2, h) || !vec(B.coef, d.act_coef, 4) || !upload(B.up, d.up_proj, B.ff, h) || !upload(B.down, d.down_proj, h, B.ff)) return bad(at + ctx->err);
            z_cols = std::max(z_cols, B.ff);
            m_cols = std::max(m_cols, B.ff);
        }
        if (c.side_dim > 0 && (!vec(B.side_norm, d.side_norm, h) || !upload(B.side_gate, d.side_gate, c.side_dim, h) || !upload(B.side_proj, d.side_proj, h, c.side_dim)))
            return bad(at + ctx->err);
    }
    b->zs = pad8(z_cols);
    b->ls = pad8(logit_cols);
    auto act = [&](void *&p, uint32_t cols) { uint8_t *q = nullptr; const bool ok = dev_alloc(e, q, act_bytes(b->f32, MB, cols)); p = q; return ok; };
    uint8_t *q = nullptr;
    if (!upload(b->head, *head, c.vocab_size, h) || !vec(b->final_norm, final_norm, h) || !dev_alloc(e, b->embed, (size_t)c.vocab_size * h, embed_bf16) ||
        (side_embed_bf16 && !dev_alloc(e, b->side_embed, (size_t)c.vocab_size * c.side_dim * n_blocks, side_embed_bf16)) ||
        !dev_alloc(e, b->x, (size_t)MB * b->hs) || !dev_alloc(e, b->z, (size_t)MB * b->zs) || !dev_alloc(e, b->proj, (size_t)MB * b->hs) || !dev_alloc(e, b->logit, (size_t)MB * b->ls) ||
        !dev_alloc(e, b->rec, rec_floats) || !dev_alloc(e, b->scan_o, (size_t)MB * o_floats) || !act(b->act_x, h) || !act(b->act_m, m_cols) || !act(b->act_s, s_cols) ||
        !dev_alloc(e, q, (size_t)MB * q_elems * (bits / 8)) || !dev_alloc(e, e->logits, (size_t)MB * c.vocab_size) || !dev_alloc(e, e->d_token, MB) || !dev_alloc(e, e->d_pos, 1) ||
        !dev_alloc(e, e->d_step, 1) || !dev_alloc(e, e->d_history, c.max_seq_len) || !dev_alloc(e, e->d_dbg, 32) || !dev_alloc(e, e->argmax_scratch, ARGMAX_SCRATCH_WORDS) ||
        !cuda_ok(ctx, cudaStreamSynchronize(ctx->stream), "engine_create_blocks"))
        return bad(ctx->err);
    b->q = q;
    e->mega_why = "block models are served by the per-operator path";
    return e;
}
