// Element-wise gated recurrences over ragged lanes with slot-held state (minGRU): every channel carries one f32 number.
#pragma once
#include "row_types.cuh"

namespace mk {

// z = sigmoid(y[z_col + c] + z_bias[c]);  u = y[x_col + c] + x_bias[c];  candidate = u >= 0 ? u + 1/2 : sigmoid(u)
// S <- (1 - z) S + z candidate;  image[t][c] = S * silu(y[g_col + c])
// State: [slot halves][width] f32.
struct MinGruArgs {
    StateLanes lanes;
    int width = 0;
    Shares y;
    int z_col = 0, x_col = 0, g_col = 0;
    const float* z_bias = nullptr;
    const float* x_bias = nullptr;
    float* state = nullptr;
    RowImage image;
    int longest = 0;  // tokens of the longest lane
};
void launch_mingru_scan(const MinGruArgs& a, cudaStream_t s);

}  // namespace mk
