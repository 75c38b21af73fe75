// Latent attention over a paged cache of one vector per token: every head's keys and values are linear in the cached vector, so
// with the queries taken to the latent space (q W_uk) all heads attend to the same rows, which serve as keys and as values, and
// what comes out is a latent per head that W_uv turns into the head's output.  Nothing but the vectors is cached.
// Tokens that come many at a time can have their keys and values expanded instead (expand helpers below) and run through the
// ordinary attention kernels.
#pragma once
#include "row_types.cuh"
#include <vector>

namespace mk {

struct LatentAttnArgs {
    const __half* q_h = nullptr;     // [n_rows][heads][rank] f16 (tensor-core kernel), or
    const float* q_f = nullptr;      // the same in f32 (general kernel)
    const void* pool = nullptr;      // [blocks * block_tokens][rank]
    int pool_f16 = 1;
    const uint32_t* tables = nullptr;
    // work list, 8 ints each, 32-byte aligned: (query row, share, n_shares, last visible position, table offset, packed row,
    // first entry of the query row, 0)
    const int32_t* entries = nullptr;
    int n_entries = 0, n_rows = 0;
    int heads = 0, rank = 0;         // rank: columns of a page row, padding included
    int block_tokens = 16;
    float scale = 1.f;
    Shares gate;                     // a head's output is multiplied by sigmoid(gate[packed row][gate_col + head])
    int gate_col = 0;
    RowImage out;                    // row head * n_rows + query row, ld = rank
    // shares (tensor-core kernel): unnormalised partial outputs [entry][heads padded][rank], (max, sum) pairs, and
    // counters [entries][CTAs per entry] that are zero before the first call and after every call
    float* part_o = nullptr;
    float* part_ml = nullptr;
    int32_t* counters = nullptr;
    int32_t* status = nullptr;       // receives a non-zero code when a bounded wait gave up
};

// The tensor-core kernel's rank for a latent of `kv_rank` values (a multiple of 128 up to 512), or 0 when it does not cover the
// case.
int latent_tc_rank(int kv_rank, int block_tokens);
// Heads of one CTA of the tensor-core kernel, and CTAs per work item.
int latent_tc_heads(int heads);
inline int latent_tc_groups(int heads) { return (heads + latent_tc_heads(heads) - 1) / latent_tc_heads(heads); }
constexpr int kLatentMaxRank = 1024;  // of the general kernel

// Host-side work list: one entry per token of lane i with n_tokens[i] < wide_from, cut into key shares while that fills the GPU.
// `rows` receives the packed rows in entry order.
struct LatentPlan {
    std::vector<int32_t> entries, rows;
    int n_entries() const { return (int)entries.size() / 8; }
    int n_rows() const { return (int)rows.size(); }
};
void plan_latent_attention(const int32_t* start_pos, const int32_t* n_tokens, const int32_t* n_blocks, int lanes, int ctas, int wide_from,
                           bool shares, LatentPlan& plan);
// Upper bounds for a tick of at most `tokens` tokens: entries, and entries with partial results.
int latent_max_entries(int tokens, int ctas);
int latent_max_shared_entries(int ctas);

void launch_latent_attention(const LatentAttnArgs& a, cudaStream_t s);

// out[r][c] = bf16(pool row of key r), r < blocks * block_tokens: the cached vectors of the listed blocks as a matmul input.
void launch_latent_gather(const void* pool, int pool_f16, const int32_t* blocks, int n_blocks, int block_tokens, int rank, __nv_bfloat16* out, cudaStream_t s);
// out[part][i][c] = bf16(x[rows[i]][part * width + c]): chosen rows cut into parts, a matmul input per part.
void launch_split_rows(const float* x, int ldx, const int32_t* rows, int n_rows, int parts, int width, __nv_bfloat16* out, cudaStream_t s);

}  // namespace mk
