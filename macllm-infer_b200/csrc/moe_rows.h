// Mixtures of experts over dense matrices: sigmoid routing, rows grouped by expert, and one gate per token for a shared expert.
#pragma once
#include "row_types.cuh"

namespace mk {

// Where the rows of a routed tick are.  A token's j-th choice is pair t * k + j.
struct MoeRows {
    int32_t* sel = nullptr;          // [T * k] expert of a pair
    float* weight = nullptr;         // [T * k] its weight
    int32_t* rank = nullptr;         // [T * k] its place among its expert's pairs
    int32_t* count = nullptr;        // [2][counts] pairs of an expert; both halves zero before the first tick
    int counts = 0;
    int32_t* offsets = nullptr;      // [experts + 1] first grouped row of an expert
    int32_t* pos_of_pair = nullptr;  // [T * k] grouped row of a pair
    float* weight_of_pos = nullptr;  // [T * k] weight of a grouped row
    float* shared_gate = nullptr;    // [T] sigmoid of logit column `experts`; null: there is none
};

// The k largest of `experts` sigmoid scores of every token (ties: the lower expert first), as they are; every pair gets a place
// among its expert's.  `half` alternates from call to call: the other half of the counts is zeroed by launch_moe_gather.
// A token with a non-finite logit leaves kMoeRouteStatus | (token & 0xFFFF) in *status; its choices stay in range.
// Either the logits are given, or the router rows w [experts (+ 1)][x.ld] (bfloat16, or f32 for f32 rows x) to be multiplied first:
// for ticks of a few rows.
void launch_moe_route(const Shares& logits, int T, int experts, int k, const MoeRows& rows, int half, int32_t* status, cudaStream_t s);
bool moe_router_is_narrow(int T, int experts, int cols);
void launch_moe_router(const RowImage& x, const void* w, int T, int experts, int k, const MoeRows& rows, int half, int32_t* status, cudaStream_t s);

// out[pos_of_pair[p]] = x[p / k] and weight_of_pos[pos_of_pair[p]] = weight[p]: rows of `bytes` bytes (a multiple of 16).
void launch_moe_gather(const void* x, int T, int experts, int k, int64_t bytes, const MoeRows& rows, int half, void* out, cudaStream_t s);

}  // namespace mk
