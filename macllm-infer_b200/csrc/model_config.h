// What a model is loaded with: the KV geometry of the reference's ModelLoadConfig (src/runtime.rs:18-91) and the choices of
// this backend.
#pragma once
#include <cstdint>

namespace mk {

struct ModelConfig {
    int device = 0;
    int block_tokens = 16, slab_blocks = 8;
    int64_t kv_capacity_tokens = 4096, prefix_capacity_tokens = 0;
    bool kv_f16 = true;
    int max_batch_tokens = 2048, max_batch_lanes = 64;
    // 0 auto (integer GEMV for a few rows, in-kernel dequant GEMM for tens of rows, f16-image GEMM for wide
    // ticks when the image fits), 1 integer GEMV only, 2 in-kernel dequant GEMM whenever the shape allows,
    // 3 f16-image GEMM whenever more than 8 rows share a matrix, 4 like 0 but nothing falls back to the in-kernel
    // dequant GEMM (f16 images for wide ticks, streamed Q4_K / Q6_K blocks for 1..64 rows)
    int matmul_path = 0;
    // expert parallelism of a sparse-MoE model: this process holds experts [ep_rank, ep_rank + 1) * experts / ep_size
    // and exchanges per-layer partial sums with the other ranks; ep_size <= 1 keeps every expert here
    int ep_rank = 0, ep_size = 1;
    // 0: all ranks run the same ticks on the same tokens (partial sums exchanged); 1: every rank schedules its own
    // sequences and each MoE layer sends the routed rows to the experts' ranks and the outputs back (ep_dispatch.cu)
    int ep_mode = 0;
    // models with recurrent layers: sequences that may be live at a time (0 = max_batch_lanes)
    int state_slots = 0;
    // dense checkpoints: 16-bit matrix operands, or everything in 32-bit (f32 matrices, activations and K/V pages)
    bool compute_f32 = false;
};

}  // namespace mk
