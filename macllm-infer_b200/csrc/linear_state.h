// Linear-attention recurrences over ragged lanes with slot-held state: WKV time mixing (a decay per key channel and a bonus for
// the current token) and the gated delta rule (one decay per head, grouped query / key heads).  State layout per slot half:
// [heads][value columns][KD] f32, value-major, KD = the key dimension padded to 32, 64, 128 or 256 - a column's keys are
// contiguous, so a decode tick streams the state with 16-byte accesses.
#pragma once
#include "row_types.cuh"

namespace mk {

// The padded key dimension of the state (throws above 256).
int linear_state_key_pad(int dim);

// What both share.  With `image` set the kernel also finishes the mixer's output - each head's row divided by its root mean
// square, times norm_w, times silu(gate) - and writes the next matmul's input; otherwise the raw rows go to `out`.
struct LinearStateArgs {
    StateLanes lanes;
    float* state = nullptr;
    int heads = 0, dim = 0, vdim = 0;
    float* out = nullptr;            // [rows][heads * vdim]
    RowImage image;                  // [rows][heads * vdim]
    const float* norm_w = nullptr;   // [heads * vdim], or [vdim] shared by the heads
    int norm_per_head = 0;           // norm_w has its own part for every head
    float eps = 0.f;
    Shares gate;                     // column gate_col + head * vdim + v
    int gate_col = 0;
};

// o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T
struct WkvScanArgs {
    LinearStateArgs common;
    Shares rkv;                      // columns r_col / k_col / v_col + head * dim + i
    int r_col = 0, k_col = 0, v_col = 0;
    const float* decay = nullptr;    // [rows][heads * dim]
    const float* bonus = nullptr;    // [heads * dim]
};
void launch_wkv_scan(const WkvScanArgs& a, cudaStream_t s);

// S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
struct DeltaScanArgs {
    LinearStateArgs common;
    int kv_heads = 0;                // head h reads query / key head h / (heads / kv_heads)
    const float* q = nullptr;        // [rows][kv_heads * dim]
    const float* k = nullptr;
    const float* v = nullptr;        // [rows][heads * vdim]
    const float* decay = nullptr;    // [rows][heads]
    const float* beta = nullptr;     // [rows][heads]
};
void launch_delta_scan(const DeltaScanArgs& a, cudaStream_t s);

// Whether the finishing form (LinearStateArgs::image) exists for these sizes.
bool linear_state_can_finish(int dim, int vdim);
// The finishing step by itself, over the raw rows in a.out.
void launch_head_norm_gate(const LinearStateArgs& a, int rows, cudaStream_t s);

}  // namespace mk
