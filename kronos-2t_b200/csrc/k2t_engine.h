// The engine object behind KronosCudaEngine and what its translation units share: k2t_engine.cu (quantized Llama/Qwen layers,
// the entry points of the C ABI, graphs, the prompt and greedy loops) and k2t_blocks.cu (models described block by block).
#pragma once
#include <algorithm>
#include <string>
#include <utility>
#include <vector>

#include "k2t_context.h"
#include "k2t_decode_mega.h"
#include "k2t_model_kernels.h"
#include "k2t_tp.h"

namespace k2t { struct BlockModel; }

struct EngineLayer {
    float *input_norm = nullptr, *post_norm = nullptr, *qkv_bias = nullptr, *q_norm = nullptr, *k_norm = nullptr;
    KronosCudaMatrix *qkv = nullptr, *o = nullptr, *gate_up = nullptr, *down = nullptr;
    // sparse-MoE FFN (router + expert records) instead of gate_up / down
    bool moe = false;
    float *router_w = nullptr, *router_bias = nullptr;
    k2t::DeviceMatrix gu_dm{}, dn_dm{};                                // geometry (and image base) of the first expert this rank holds: template of the expert launches
    uint8_t *d_experts = nullptr;                                     // ONE allocation: the device images of all experts of the layer this rank holds
    const uint8_t **d_gu_bases = nullptr, **d_dn_bases = nullptr;     // device tables: image base of every expert
    k2t::ExpertCodebook *d_gu_books = nullptr, *d_dn_books = nullptr; // device tables: decode tables of every expert
    int gu_fmt = -1, dn_fmt = -1;                                     // kernel format of the layer's experts
    uint32_t expert0 = 0;                                             // first expert held by this rank (expert parallelism)
    uint32_t *d_route_ids = nullptr;                                  // [max_batch][32] routes of the last batch
    float *d_route_w = nullptr;
    // shared expert of a MoE layer (SharedMoeExpert, sparse_moe.rs:223-315): its matrices live in gate_up / down above
    uint32_t sh_inter = 0;
    float *sh_gate_w = nullptr;
};

struct KronosCudaEngine {
    KronosCudaContext *ctx = nullptr;
    KronosCudaEngineConfig cfg{};
    std::vector<EngineLayer> layers;
    KronosCudaMatrix *lm_head = nullptr;
    float *final_norm = nullptr, *rope = nullptr;
    uint16_t *embed_bf16 = nullptr;
    // workspace
    float *hidden = nullptr, *proj = nullptr, *qkv = nullptr, *gate_up = nullptr, *logits = nullptr;
    int8_t *act_q = nullptr, *q_i8 = nullptr;
    float *attn_tap = nullptr;                // attention output of the last layer (diagnostic)
    float *act_s = nullptr, *q_scale = nullptr, *part_m = nullptr, *part_l = nullptr, *part_o = nullptr;
    float *attn_sc = nullptr, *attn_bmax = nullptr;      // long contexts in CPU order: scores [n_q][kv_stride], block maxima [n_q][kv_stride / 128]
    bool split_kv = false;                    // long contexts by the split-KV kernels instead (config flag, or the cache is too long for the exact path)
    int32_t *act_m = nullptr;
    int8_t *k_q8 = nullptr, *v_q8 = nullptr;
    int8_t *v_t = nullptr;      // int8 cache without a window: the value rows once more, transposed in 16-position blocks for the value chains
    float *k_scale = nullptr, *v_scale = nullptr;
    uint32_t *d_token = nullptr, *d_pos = nullptr, *d_step = nullptr, *d_history = nullptr;
    uint32_t n_split = 32;
    uint32_t max_batch = 256;                 // tokens per prompt batch: their projections run on the tensor cores in one weight pass (k2t_gemm_tc.cu), their attention side by side; every per-token buffer holds this many rows (KRONOS_CUDA_PROMPT_BATCH, 16..512)
    uint32_t ctx_bound = 0;                   // prompt batches (launched eagerly, position known on the host): no token of the batch sees more positions; 0 = size launches for the whole cache
    uint32_t kv_stride = 0;                   // cache rows per (layer, kv head): the rows the geometry needs (max_seq_len, or sinks + ring) rounded up to 32, so every 32-row tile of rows and scales starts on 16 bytes
    k2t::KvRing ring{};                       // sliding-window + sink ring (all zero: row = position)
    uint32_t kv_rows = 0;                     // rows in use per (layer, kv head)
    // sparse-MoE workspace: normalised hidden state, per-route expert buffers
    float *x_norm = nullptr, *moe_gu = nullptr, *moe_out = nullptr, *router_logits = nullptr;
    uint32_t *router_done = nullptr;
    int8_t *moe_q = nullptr; float *moe_s = nullptr; int32_t *moe_m = nullptr;
    // shared-expert workspace, [max_batch] rows each: gate_up outputs, the down projection's activation, outputs, gate values
    uint32_t sh_inter_max = 0;
    float *sh_gu = nullptr, *sh_out = nullptr, *sh_scale = nullptr;
    int8_t *sh_q = nullptr; float *sh_s = nullptr; int32_t *sh_m = nullptr;
    bool has_moe = false;
    // tensor parallel: exchange buffer (data[2][tp][slot] floats + flags[tp]) and the peers' mappings
    k2t::TpLink tp{};
    float *tp_buf = nullptr;
    uint32_t *tp_done = nullptr;              // CTAs of the current fused exchange that have finished (device word)
    std::vector<void *> tp_peers;            // mappings opened with cudaIpcOpenMemHandle
    bool tp_ready = false;
    float *logits_local = nullptr;            // this rank's logits slice [max_batch][vocab_size]
    KronosCudaMatrix *embed_matrix = nullptr; // whole lm_head for the token lookup (tied embeddings under tp)
    uint32_t last_row = 0;                    // row of `hidden` that holds the last forwarded token (prompt batches)
    bool pdl = true;                          // kernels of a step overlap their prologues with the predecessor's tail
    bool fused = false;                       // single-token steps: norm / SwiGLU / embedding run as prologues of the GEMV that consumes them (KRONOS_CUDA_FUSED=1)
    const float *final_hidden = nullptr;      // where the last step left the residual stream of its last token
    size_t weight_bytes = 0;
    std::vector<void *> allocs;
    // whole-token decode kernel (contexts up to ATTN_EXACT_CTX positions)
    bool mega_ok = false;
    std::string mega_why;                     // why the kernel is not used, when it is not
    float *hidden2 = nullptr;
    k2t::MegaLayer *d_mega_layers = nullptr;
    k2t::MegaMatrix *d_mega_head = nullptr;
    uint32_t *d_barrier = nullptr;
    unsigned long long *d_trace = nullptr;    // phase trace of the last step of the last decode-kernel call
    uint32_t mega_warp_smem = 0, mega_kmax = 0;
    size_t mega_smem = 0;
    cudaGraphExec_t graphs[4] = {nullptr, nullptr, nullptr, nullptr};      // [greedy ? 0 : 1][long context ? 1 : 0] -> 2 * ids + long
    cudaStream_t graph_stream = nullptr;      // the stream the graphs were captured on
    // per-kernel-class timing of one step (kronos_cuda_engine_profile_step): while prof_on, every launch is followed
    // by an event record, so a captured step carries one event node per kernel
    bool prof_on = false;
    std::vector<std::pair<const char *, cudaEvent_t>> prof_marks;
#ifdef K2T_TIMELINE
    std::vector<const char *> tl_labels[4];     // launch labels of the four captured step graphs, in launch order
    std::vector<const char *> *tl_cur = nullptr;
#endif
    k2t::BlockModel *blocks = nullptr;        // set: the model is a list of blocks (k2t_blocks.h) and `layers` is not used
    unsigned long long *d_dbg = nullptr;      // 32 diagnostic words (phase clocks of the attention kernel, layer 0)
    float *argmax_scratch = nullptr;          // candidates and arrival counter of the argmax kernel
    bool attn_trace = false;
};

namespace k2t {

// what a batch leaves behind: argmax of its (single) token, logits of the last token, of all tokens, nothing
enum class Tail { Greedy, LastLogits, AllLogits, None };

// books `n` launches (and, while a step is profiled, an event behind them); false with the context's error set when err is one
bool engine_count(KronosCudaEngine *e, cudaError_t err, const char *what, uint32_t n = 1);

template <typename T>
inline bool dev_alloc(KronosCudaEngine *e, T *&p, size_t count, const T *host = nullptr) {
    void *raw = nullptr;
    const size_t bytes = std::max<size_t>(count, 1) * sizeof(T);
    if (!cuda_ok(e->ctx, cudaMalloc(&raw, bytes), "cudaMalloc(engine)")) return false;
    e->allocs.push_back(raw);
    p = static_cast<T *>(raw);
    if (host) return cuda_ok(e->ctx, cudaMemcpyAsync(p, host, count * sizeof(T), cudaMemcpyHostToDevice, e->ctx->stream), "upload");
    return cuda_ok(e->ctx, cudaMemsetAsync(p, 0, bytes, e->ctx->stream), "clear");
}


inline void dev_free(KronosCudaEngine *e, void *p) {
    if (!p) return;
    for (size_t i = 0; i < e->allocs.size(); ++i)
        if (e->allocs[i] == p) { e->allocs.erase(e->allocs.begin() + i); break; }
    cudaFree(p);
}

}  // namespace k2t
