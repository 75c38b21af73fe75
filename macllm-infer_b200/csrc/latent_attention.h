// Latent attention over a paged cache of one vector per token: every head's keys and values are linear in the cached vector, so
// with the queries taken to the latent space (q W_uk) all heads attend to the same rows, which serve as keys and as values, and
// what comes out is a latent per head that W_uv turns into the head's output.  Nothing but the vectors is cached.
// A row of the cache may hold more columns than the vector: a key part that all heads share, cached as it is after its rotation,
// which counts in the scores only.  The queries' part of it arrives before its rotation and turns while it is read.
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
    int values = 0;                  // columns of the output: the vector's, padding included (0: rank)
    // queries' columns rot0 .. rot0 + rot_dims - 1 turn in adjacent pairs; rot0 a multiple of 8, tables [positions][rot_dims / 2]
    int rot0 = 0, rot_dims = 0;
    const float *cos_t = nullptr, *sin_t = nullptr;
    int window = 0;                  // a position sees itself and the window - 1 keys before it; 0: all before it
    const float* sink = nullptr;     // [heads]: one more term exp(sink) in the denominator; null: none
    int block_tokens = 16;
    float scale = 1.f;
    Shares gate;                     // a head's output is multiplied by sigmoid(gate[packed row][gate_col + head]); no pointer: it is not
    int gate_col = 0;
    RowImage out;                    // row head * n_rows + query row, ld = values
    // shares (tensor-core kernel): unnormalised partial outputs [entry][heads padded][values], (max, sum) pairs, and
    // counters [entries][CTAs per entry] that are zero before the first call and after every call
    float* part_o = nullptr;
    float* part_ml = nullptr;
    int32_t* counters = nullptr;
    int32_t* status = nullptr;       // receives a non-zero code when a bounded wait gave up
};

// The tensor-core kernel's columns for a vector of `kv_rank` values with a shared key part of `rot_width` (0: none), which begins at
// column rot0: of the values (a multiple of 128 up to 512) and of a page row (a multiple of 64, at most 128 more).
struct LatentColumns {
    int values = 0, row = 0, rot0 = 0;  // row = 0: it does not cover the case
};
LatentColumns latent_tc_columns(int kv_rank, int rot_width, int block_tokens);
// The same of the general kernel.
LatentColumns latent_general_columns(int kv_rank, int rot_width);
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
                           bool shares, LatentPlan& plan, int window = 0);
// Upper bounds for a tick of at most `tokens` tokens: entries, and entries with partial results.
int latent_max_entries(int tokens, int ctas);
int latent_max_shared_entries(int ctas);

void launch_latent_attention(const LatentAttnArgs& a, cudaStream_t s);

// out[r][c] = bf16(pool row of key r), r < blocks * block_tokens: the cached vectors of the listed blocks as a matmul input.
void launch_latent_gather(const void* pool, int pool_f16, const int32_t* blocks, int n_blocks, int block_tokens, int rank, __nv_bfloat16* out, cudaStream_t s);
// out[part][i][c] = bf16(x[rows[i]][part * width + c]): chosen rows cut into parts, a matmul input per part.
void launch_split_rows(const float* x, int ldx, const int32_t* rows, int n_rows, int parts, int width, __nv_bfloat16* out, cudaStream_t s);

}  // namespace mk
