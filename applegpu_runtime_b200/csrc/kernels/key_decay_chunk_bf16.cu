// The chunked form of key-decayed matrix states for bfloat16 storage (a file per type, so that they compile side by side).
#include "key_decay_chunk.cuh"

namespace ag { namespace k {

Status key_decay_chunked_bf16(cudaStream_t s, const KdParams& p) { return launch_chunked<__nv_bfloat16>(s, p); }

}}  // namespace ag::k
