// Mixtures of experts over dense matrices: sigmoid routing, rows grouped by expert, and one gate per token for a shared expert.
#pragma once
#include "row_types.cuh"

namespace mk {

// Where the rows of a routed tick are.  A token's j-th choice is pair t * k + j.
struct MoeRows {
    int32_t* sel = nullptr;          // [T * k] expert of a pair
    float* weight = nullptr;         // [T * k] its weight
    int32_t* offsets = nullptr;      // [experts + 1] first grouped row of an expert
    int32_t* pos_of_pair = nullptr;  // [T * k] grouped row of a pair
    int32_t* token_of_pos = nullptr; // [T * k]
    float* weight_of_pos = nullptr;  // [T * k] weight of a grouped row
    float* shared_gate = nullptr;    // [T] sigmoid of logit column `experts`; null: there is none
};

// The k largest of `experts` sigmoid scores of every token (ties: the lower expert first), as they are, and the pairs grouped by
// expert.  A token with a non-finite logit leaves kMoeRouteStatus | (token & 0xFFFF) in *status; its choices stay in range.
// Returns the number of kernels launched.
int launch_moe_rows(const Shares& logits, int T, int experts, int k, const MoeRows& rows, int32_t* status, cudaStream_t s);

// out[pos_of_pair[p]] = x[p / k] and weight_of_pos[pos_of_pair[p]] = weight[p]: rows of `bytes` bytes (a multiple of 16).
void launch_moe_gather(const void* x, int T, int k, int64_t bytes, const MoeRows& rows, void* out, cudaStream_t s);

}  // namespace mk
