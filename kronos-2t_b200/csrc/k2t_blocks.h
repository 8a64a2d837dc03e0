// Models described block by block (kronos_cuda_engine_create_blocks): what k2t_engine.cu calls of k2t_blocks.cu.
#pragma once
#include "k2t_engine.h"

namespace k2t {

// queues the kernels of T consecutive tokens (see enqueue_batch)
bool blocks_enqueue(KronosCudaEngine *e, uint32_t T, bool embed, Tail tail);
uint32_t blocks_step_launches(const KronosCudaEngine *e);
// A forward call from position `pos`: 0 starts a sequence (recurrent state cleared); otherwise the sequence must stand there.
// Between begin and end the sequence counts as lost, so a call that fails half-way is followed by a restart at 0.
bool blocks_begin(KronosCudaEngine *e, bool token_ids, size_t pos);
void blocks_end(KronosCudaEngine *e, size_t pos);
bool blocks_can_continue(const KronosCudaEngine *e, size_t pos);
// puts the recurrent state aside (save) and back, around steps whose results do not count
bool blocks_park_state(KronosCudaEngine *e, bool save);
size_t blocks_kv_bytes(const KronosCudaEngine *e, size_t positions);
size_t blocks_snapshot_bytes(const KronosCudaEngine *e);
bool blocks_save(KronosCudaEngine *e, size_t n, size_t cur_pos, uint8_t *out);
bool blocks_restore(KronosCudaEngine *e, const uint8_t *data, size_t len);
const float *blocks_hidden(const KronosCudaEngine *e);
void blocks_destroy(KronosCudaEngine *e);

}  // namespace k2t
