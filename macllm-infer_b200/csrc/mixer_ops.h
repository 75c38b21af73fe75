// The steps between the matmuls of mixer-built decoders: residual update with norm and token shift or short convolution, the decay
// of WKV time mixing, the short convolution and unit norms of the gated delta rule, the channel gates of the other delta rule,
// output gates, the per-layer token input - and the 32-bit matmul for models computed in f32 throughout.
#pragma once
#include "mixer_spec.h"
#include "device_util.h"
#include "row_types.cuh"

namespace mk {

// One CTA per row r (x row = row_index ? row_index[r] : r):
//   x_out = x + coef * sum over branches b of (add_w[b] ? rms(add[b]) * add_w[b] : add[b])      (n_add branches; x = 0 when null)
//   (a single branch may carry a bias [width], added before its norm; a single normed branch also the rows of the experts a token
//    chose, added up before its norm - its own matrix may then be missing)
//   raw    <- x_out                        (optional image)
//   h       = norm(x_out);  normed <- h    (optional image, n_mix = 0)
//   mixes[i] <- h + (h' - h) * mu[i]       (n_mix images of `rows` rows each, one after the other), h' = h of the sequence's
//                                          previous token: recomputed from the row before, or the kept one (zeros at the start)
// The last row of every lane leaves its h as the kept one.  x and x_out are different buffers when n_mix > 0, because a row
// reads its neighbour's old value.
struct RowUpdateArgs {
    const float* x = nullptr;
    float* x_out = nullptr;  // may be null (nothing kept)
    int rows = 0, width = 0;
    const int32_t* row_index = nullptr;
    int n_add = 0;
    Shares add[2];
    const float* add_w[2] = {nullptr, nullptr};
    const float* add_bias = nullptr;
    const float* routed = nullptr;       // [rows of all experts][width]
    const int32_t* routed_at = nullptr;  // [token][routed_k]: where a token's rows are
    int routed_k = 0;
    float add_coef = 1.f, add_eps = 0.f;
    RowImage raw;
    NormKind norm = NormKind::None;
    float alpha = 1.f;          // DynTanh
    float norm_eps = 0.f;       // Layer, Rms
    const float* norm_w = nullptr;
    const float* norm_b = nullptr;  // DynTanh
    RowImage normed;
    int n_mix = 0;
    const float* mu = nullptr;  // [n_mix][width]
    RowImage mixes;
    StateLanes lanes;
    const int32_t* token_lane = nullptr;
    float* kept = nullptr;      // [slot halves][width]
    // taps > 0:  normed <- h + sum_j conv[j] h of the row taps - 1 - j before (zeros before the sequence's start), the rows' norm
    // recomputed like the token shift's; `kept` then holds the last taps - 1 rows, [slot halves][taps - 1][width].  At most one
    // un-normed branch; an RMS norm.
    int taps = 0;
    const float* conv = nullptr;  // [taps][width]
};
void launch_row_update(const RowUpdateArgs& a, cudaStream_t s);

// decay[t][c] = exp(-exp(sum_j tanh(low[t][j]) w2[c][j] + w0[c])), everything in f32.  w2t is w2 transposed, [rank][channels].
void launch_wkv_decay(const Shares& low, int low_col, int rows, int rank, int channels, const float* w2t, const float* w0, float* decay, cudaStream_t s);

// What the delta rule with channel gates needs beside its projections, everything in f32, per row of the lanes and key channel c of a head:
//   decay   = exp(-exp(-1/2) sigmoid(sum_j tanh(y[low_col + j]) w2[c][j] + w0[c]))
//   removal = sigmoid(y[a_col + c] + a_bias[c]) k[c] / (sum of the head's k^2 + 1e-6),  k = y[k_col + c]
struct ChannelGatesArgs {
    Shares y;
    int k_col = 0, a_col = 0, low_col = 0;
    StateLanes lanes;
    int longest = 0;                // rows of the longest lane
    int heads = 0, dim = 0, rank = 0;
    const float* w2t = nullptr;     // w2 transposed, [rank][heads * dim]
    const float* w0 = nullptr;      // [heads * dim]
    const float* a_bias = nullptr;  // [heads * dim]
    float* decay = nullptr;         // [rows][heads * dim]
    float* removal = nullptr;
};
void launch_channel_gates(const ChannelGatesArgs& a, cudaStream_t s);

// The gated delta rule's inputs from the raw projections y: a causal convolution of `taps` taps per channel over q | k | v and
// silu, unit norm per head of q and k (q also times dim^-1/2), beta = sigmoid(b), decay = exp(softplus(a + dt_bias) * log_decay).
// The kept tail is the last taps - 1 raw rows of a sequence, [slot halves][taps - 1][channels] over q | k | v.
struct DeltaPrepArgs {
    Shares y;
    int q_col = 0, k_col = 0, v_col = 0, a_col = 0, b_col = 0;
    int rows = 0, heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 1;
    const float* conv = nullptr;       // [taps][channels] over q | k | v
    const float* dt_bias = nullptr;    // [heads]
    const float* log_decay = nullptr;  // [heads], negative
    StateLanes lanes;
    const int32_t* token_lane = nullptr;
    float* tail = nullptr;
    float *q = nullptr, *k = nullptr, *v = nullptr, *beta = nullptr, *decay = nullptr;
};
void launch_delta_prep(const DeltaPrepArgs& a, cudaStream_t s);

// out[t][h * vdim + i] = attn[t][h * row_width + i] * sigmoid(gate[t][gate_col + h]), t = row_list[0 .. rows) or 0 .. rows - 1
// (OutputGate::Value: sigmoid(gate[t][gate_col + h * vdim + i]); None: no factor), all of it times `scale`
void launch_head_gate(const float* attn, int rows, int heads, int row_width, int vdim, const Shares& gate, int gate_col, const RowImage& out,
                      cudaStream_t s, const int32_t* row_list = nullptr, OutputGate kind = OutputGate::Head, float scale = 1.f);

// out[t][j] = gelu_tanh(z[t][j]) * table[ids[t]][slice + j], j < dim; table [vocab][table_ld] as bfloat16 bits (or f32)
void launch_side_gate(const Shares& z, int rows, int dim, const uint32_t* ids, const void* table, int table_f32, int64_t table_ld, int slice,
                      const RowImage& out, cudaStream_t s);

// out[t][j] = act(gu[t][2j], gu[t][2j + 1]), j < ff: gate and up rows interleaved
void launch_gated_act(const Shares& gu, int rows, int ff, const RowImage& out, cudaStream_t s, const GatedAct& act = {});

// y[t][n] = sum_k x[t][k] w[n][k] in f32, k ascending.  x is [n_groups][T][cols]; weight row n reads input g of its group, whose
// rows end at 128 * group_end[g], or are 128 * group_tiles each (see HalfWeight).  `to` scatters the result instead (see
// MatmulScatter).  The result is multiplied by `scale` and, with a soft cap c, becomes c * tanh(y / c).
void launch_f32_matmul(const float* w, int64_t rows, int cols, const float* x, int T, float* y, int ldy, int n_groups, const int* group_end,
                       cudaStream_t s, int group_tiles = 0, float scale = 1.f, const MatmulScatter* to = nullptr, float softcap = 0.f);
// The same over rows grouped by expert: rows [offsets[e], offsets[e + 1]) of x and y meet matrix e of `experts`, rows x cols each,
// matrix_rows apart.  T: rows of all experts.
void launch_f32_matmul_experts(const float* w, int experts, const int32_t* offsets, int64_t rows, int64_t matrix_rows, int cols, const float* x, int T, float* y,
                               int ldy, cudaStream_t s);

// The embedding output of models with sinusoidal positions:  e = table[ids[t]] + sinusoid(positions[t]);  x = layer norm of e, in
// f32 to x [rows][width] and as a matmul input to `image` (optional).  freq[i] is the frequency of column pair i in f64: the angle
// of a far position is as exact as that of a near one.
struct EmbedNormArgs {
    const uint32_t* ids = nullptr;
    const int32_t* positions = nullptr;
    const void* table = nullptr;  // [vocab][width] bfloat16 bits, or f32
    int table_f32 = 0;
    int rows = 0, width = 0;
    const double* freq = nullptr;  // [ceil(width / 2)]
    const float* norm_w = nullptr;
    float eps = 0.f;
    float* x = nullptr;
    RowImage image;
};
void launch_embed_norm(const EmbedNormArgs& a, cudaStream_t s);

// What a row's projections need before the next matmuls, one CTA per (row, part):
//   part 1 (q_rank > 0): the query latent RMS-normed into q_image, the key/value latent RMS-normed into its page; behind it, at
//                        column rot0, the shared key part of rot_width columns, whose first rot_dims turn in adjacent pairs
//   part 2 (ff > 0):     poly = a N(z) + b N(z^2) + c N(z^3) + e over z = y[ff_col ..] + ff_bias, N = division by the row's root
//                        mean square
struct LatentPrepArgs {
    Shares y;
    int rows = 0;
    float eps = 0.f;
    int q_col = 0, q_rank = 0;
    const float* q_norm = nullptr;
    RowImage q_image;
    int kv_col = 0, kv_rank = 0, kv_width = 0;  // kv_width: columns of a page row, the rest is zeros
    const float* kv_norm = nullptr;
    const int64_t* slots = nullptr;
    void* pool = nullptr;                       // [blocks * block_tokens][kv_width]
    int pool_f16 = 1;
    int rot_col = 0, rot0 = 0, rot_width = 0, rot_dims = 0;
    const float *cos_t = nullptr, *sin_t = nullptr;  // [positions][rot_dims / 2]
    const int32_t* positions = nullptr;
    int lat_vec = 0;                            // the latents lie in whole 16-byte packs (filled in by the launcher)
    int ff_col = 0, ff = 0;
    const float* ff_bias = nullptr;
    const float* poly = nullptr;                // [4]
    RowImage ff_image;
};
void launch_latent_prep(const LatentPrepArgs& a, cudaStream_t s);

}  // namespace mk
