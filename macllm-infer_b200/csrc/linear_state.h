// Linear-attention recurrences over ragged lanes with slot-held state: WKV time mixing (a decay per key channel and a bonus for
// the current token), the gated delta rule (one decay per head, grouped query / key heads), the matrix memory of mLSTM (one
// decay per head from exponential gates, a normaliser) and the delta rule with a decay and a removal rate per key channel.  State layout per slot half: [heads][value columns][KD] f32, value-major,
// KD = the key dimension padded to 32, 64, 128 or 256 - a column's keys are contiguous, so a decode tick streams the state with
// 16-byte accesses.  mLSTM has one column more than values: the normaliser, whose value is always 1.
#pragma once
#include "row_types.cuh"

namespace mk {

// The padded key dimension of the state (throws above 256).
int linear_state_key_pad(int dim);

// What all share.  With `image` set the kernel also finishes the mixer's output - each head's row divided by its root mean
// square, times norm_w, times silu(gate) or sigmoid(gate) - and writes the next matmul's input; otherwise the raw rows go to `out`.
struct LinearStateArgs {
    StateLanes lanes;
    float* state = nullptr;
    int heads = 0, dim = 0, vdim = 0;
    float* out = nullptr;            // [rows][heads][vdim], normalised: [rows][heads][linear_state_raw_width(vdim)]
    int normalised = 0;              // a raw head row ends with its denominator (mLSTM): divided by it before the norm
    int gate_sigmoid = 0;            // sigmoid(gate) instead of silu(gate)
    float out_scale = 1.f;           // of the finished rows
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

// Raw row of a normalised head: its values, then the denominator.
__host__ __device__ inline int linear_state_raw_width(int vdim) { return (vdim + 4) / 4 * 4; }

// Per head: i = cap tanh((zi + i_bias) / cap), f = log sigmoid(cap tanh((zf + f_bias) / cap));
// m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T, n likewise with k alone, m <- m' (0 at the start);
// o = S^T q / (max(|n . q|, exp(-m)) + 1e-6), q times dim^-1/2.
struct MlstmScanArgs {
    LinearStateArgs common;
    Shares y;                        // columns q_col / k_col + head * dim + i, v_col + head * vdim + v, i_col / f_col + head
    int q_col = 0, k_col = 0, v_col = 0, i_col = 0, f_col = 0;
    const __nv_bfloat16* yh = nullptr;  // q, k and v come from these rows [rows][ldh] instead (16-byte aligned, ldh a multiple of 8):
    int ldh = 0;                        // what the chunked form reads
    const float* i_bias = nullptr;   // [heads]
    const float* f_bias = nullptr;
    float cap = 1.f;
    float* running_max = nullptr;    // [slot halves][heads]
    int32_t* counters = nullptr;     // [lanes][heads], zero before the first call; every call leaves them zero
    int rows = 0, longest = 0;       // of all lanes, of the longest one
    int rounded = 0;                 // queries, keys and values are rounded to bfloat16 (as the chunked form has them)
};
// One-token lanes, prompts in chunks (yh set), prompts row by row in f32 (otherwise).  Always finishes (common.image is set,
// common.out is scratch).  Returns the number of kernels launched.
int launch_mlstm_scan(const MlstmScanArgs& a, cudaStream_t s);
// The forms behind it (mlstm.cu): one-token lanes, finished; chunks of prompts, whose raw rows are [heads][vdim] and divided already.
void launch_mlstm_step(const MlstmScanArgs& a, cudaStream_t s);
void launch_mlstm_chunks(const MlstmScanArgs& a, cudaStream_t s);

// S <- diag(w) S - (a u)(u^T S) + k v^T with both terms reading the old state, u the head's unit key;  o = S^T r.  With
// removal = a k / (sum k^2 + 1e-6) the middle term is removal (k^T S).
struct ChannelDeltaArgs {
    LinearStateArgs common;
    Shares y;                        // columns r_col / k_col / v_col + head * dim + i
    int r_col = 0, k_col = 0, v_col = 0;
    const float* decay = nullptr;    // [rows][heads * dim]
    const float* removal = nullptr;  // [rows][heads * dim]
    // for the forms that make decay and removal themselves (see ChannelGatesArgs): the columns of the removal rates' and of the
    // low-rank input, and the weights; w2h: w2t as bfloat16, taken instead when it is there
    int a_col = 0, low_col = 0, rank = 0;
    const float *w2t = nullptr, *w0 = nullptr, *a_bias = nullptr;
    const __nv_bfloat16* w2h = nullptr;
};
// Row by row, from `decay` and `removal`.
void launch_channel_delta_scan(const ChannelDeltaArgs& a, cudaStream_t s);
// One-token lanes, from the projections; finishes (common.image is set).
bool channel_delta_can_step(int dim, int rank);
void launch_channel_delta_step(const ChannelDeltaArgs& a, cudaStream_t s);
// Prompts in chunks on tensor cores, from the projections (w2h is set), lanes in packed order, the longest of `longest` rows; leaves
// the raw rows in common.out.  `scratch`: channel_delta_chunk_bytes for all tokens and lanes of a tick.  Two kernels.
bool channel_delta_can_chunk(int dim);
size_t channel_delta_chunk_bytes(int dim, int heads, int tokens, int lanes);
void launch_channel_delta_chunks(const ChannelDeltaArgs& a, int longest, void* scratch, cudaStream_t s);
#ifdef __CUDACC__
// The decay of a channel from the logit of its low-rank projection, exp(-exp(-1/2) sigmoid(z)), and its logarithm.
__device__ __forceinline__ float channel_log_decay_f(float z) { return -0.60653066f * sigmoid_f(z); }
__device__ __forceinline__ float channel_decay_f(float z) { return expf(channel_log_decay_f(z)); }

// N values per lane summed over LPC lanes (a power of two): lane l ends with value(s) first .. first + returned - 1 in v[0 ..].
template <int N, int LPC>
__device__ __forceinline__ int fold_lanes(float (&v)[N], int lane, int& first) {
    int n = N;
    first = 0;
#pragma unroll
    for (int x = 1; x < LPC; x <<= 1) {
        if (n > 1) {
            n >>= 1;
            const bool up = (lane & x) != 0;
#pragma unroll
            for (int i = 0; i < N / 2; ++i)
                if (i < n) v[i] = (up ? v[i + n] : v[i]) + __shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + n], x);
            first += up ? n : 0;
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], x);
        }
    }
    return n;
}
#endif

// Whether the finishing form (LinearStateArgs::image) exists for these sizes.
bool linear_state_can_finish(int dim, int vdim);
// The finishing step by itself, over the raw rows in a.out.
void launch_head_norm_gate(const LinearStateArgs& a, int rows, cudaStream_t s);

}  // namespace mk
