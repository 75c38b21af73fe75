// See gated_scan.h.
//
// A row is an affine map S -> a S + b of every channel, so rows compose: prompts run in tiles of 128 rows, 16 channels per CTA.
// A thread folds four consecutive rows of one channel, one warp per channel then scans the 32 folded maps with shuffles, and the
// threads walk their four rows again from the state they now know.  The next tile's projections are on their way meanwhile.
// a = 1 - z lies in (0, 1) and b is what the gate lets in, so composing loses nothing but rounding.  Short lanes take a thread per
// channel that walks the rows.
#include "gated_scan.h"
#include <algorithm>

namespace mk {

namespace {

constexpr int GS_CH = 16;       // channels of a CTA
constexpr int GS_SLICES = 32;   // row slices of a tile, one per lane of the scanning warp
constexpr int GS_ROWS = 4;      // rows of a slice
constexpr int GS_TILE = GS_SLICES * GS_ROWS;
constexpr int GS_THREADS = GS_CH * GS_SLICES;
constexpr int GS_SHORT = 8;     // lanes up to this many rows are walked row by row
constexpr int GS_SHORT_THREADS = 128;

static_assert(GS_THREADS / 32 == GS_CH, "one warp scans one channel");

__device__ __forceinline__ float candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoid_f(u); }

__global__ void __launch_bounds__(GS_THREADS) mingru_wide_kernel(MinGruArgs a) {
    __shared__ float s_a[GS_CH][GS_SLICES + 1], s_b[GS_CH][GS_SLICES + 1], s_in[GS_CH][GS_SLICES + 1];
    const int ch = threadIdx.x & (GS_CH - 1), slice = threadIdx.x / GS_CH;
    const int c = blockIdx.x * GS_CH + ch;
    const bool live = c < a.width;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    const StateLane sl = a.lanes.at(blockIdx.y);
    const int wc = blockIdx.x * GS_CH + warp;  // the channel this warp scans
    float carry = sl.in >= 0 && wc < a.width ? a.state[(int64_t)sl.in * a.width + wc] : 0.f;
    const float zb = live ? a.z_bias[c] : 0.f, xb = live ? a.x_bias[c] : 0.f;
    pdl_wait();

    float pz[GS_ROWS], px[GS_ROWS], pg[GS_ROWS];
    auto fetch = [&](int tile) {
#pragma unroll
        for (int i = 0; i < GS_ROWS; ++i) {
            const int r = tile * GS_TILE + slice * GS_ROWS + i;
            if (live && r < sl.n) {
                pz[i] = a.y.at(sl.first + r, a.z_col + c);
                px[i] = a.y.at(sl.first + r, a.x_col + c);
                pg[i] = a.y.at(sl.first + r, a.g_col + c);
            }
        }
    };
    const int tiles = (sl.n + GS_TILE - 1) / GS_TILE;
    fetch(0);
    for (int t = 0; t < tiles; ++t) {
        const int r0 = t * GS_TILE + slice * GS_ROWS;
        float ka[GS_ROWS], kb[GS_ROWS], g[GS_ROWS], fa = 1.f, fb = 0.f;
#pragma unroll
        for (int i = 0; i < GS_ROWS; ++i) {
            ka[i] = 1.f;  // a row past the end changes nothing
            kb[i] = 0.f;
            g[i] = 0.f;
            if (live && r0 + i < sl.n) {
                const float z = sigmoid_f(pz[i] + zb);
                ka[i] = 1.f - z;
                kb[i] = z * candidate(px[i] + xb);
                g[i] = silu_f(pg[i]);
            }
            fb = fmaf(ka[i], fb, kb[i]);
            fa *= ka[i];
        }
        if (t + 1 < tiles) fetch(t + 1);
        s_a[ch][slice] = fa;
        s_b[ch][slice] = fb;
        __syncthreads();
        float va = s_a[warp][lane], vb = s_b[warp][lane];
#pragma unroll
        for (int x = 1; x < GS_SLICES; x <<= 1) {
            const float pa = __shfl_up_sync(0xffffffffu, va, x), pb = __shfl_up_sync(0xffffffffu, vb, x);
            if (lane >= x) {
                vb = fmaf(va, pb, vb);
                va *= pa;
            }
        }
        const float after = fmaf(va, carry, vb);                         // the state behind this lane's slice
        const float before = __shfl_up_sync(0xffffffffu, after, 1);
        s_in[warp][lane] = lane == 0 ? carry : before;
        carry = __shfl_sync(0xffffffffu, after, 31);
        __syncthreads();
        float S = s_in[ch][slice];
#pragma unroll
        for (int i = 0; i < GS_ROWS; ++i) {
            S = fmaf(ka[i], S, kb[i]);
            if (live && r0 + i < sl.n) a.image.put(sl.first + r0 + i, c, S * g[i]);
        }
    }
    if (lane == 0 && wc < a.width) a.state[(int64_t)sl.out * a.width + wc] = carry;
    // the columns that pad the image
    if (blockIdx.x == gridDim.x - 1)
        for (int r = threadIdx.x / 32; r < sl.n; r += GS_THREADS / 32)
            for (int p = a.width + lane; p < a.image.end(); p += 32) a.image.put(sl.first + r, p, 0.f);
}

__global__ void __launch_bounds__(GS_SHORT_THREADS) mingru_short_kernel(MinGruArgs a) {
    const int c = blockIdx.x * GS_SHORT_THREADS + threadIdx.x;
    const bool live = c < a.width;
    pdl_trigger();
    const StateLane sl = a.lanes.at(blockIdx.y);
    float S = live && sl.in >= 0 ? a.state[(int64_t)sl.in * a.width + c] : 0.f;
    const float zb = live ? a.z_bias[c] : 0.f, xb = live ? a.x_bias[c] : 0.f;
    pdl_wait();
    if (c >= a.image.end()) return;
    for (int r = 0; r < sl.n; ++r) {
        const int64_t row = sl.first + r;
        if (!live) {
            a.image.put(row, c, 0.f);
            continue;
        }
        const float z = sigmoid_f(a.y.at(row, a.z_col + c) + zb);
        S = fmaf(1.f - z, S, z * candidate(a.y.at(row, a.x_col + c) + xb));
        a.image.put(row, c, S * silu_f(a.y.at(row, a.g_col + c)));
    }
    if (live) a.state[(int64_t)sl.out * a.width + c] = S;
}

}  // namespace

void launch_mingru_scan(const MinGruArgs& a, cudaStream_t s) {
    if (a.lanes.lanes <= 0) return;
    if (a.lanes.lanes > 65535) throw std::runtime_error("launch_mingru_scan: at most 65535 lanes");
    if (a.longest <= GS_SHORT) {
        const dim3 grid((unsigned)((a.image.end() + GS_SHORT_THREADS - 1) / GS_SHORT_THREADS), (unsigned)a.lanes.lanes);
        launch_pdl(mingru_short_kernel, grid, dim3(GS_SHORT_THREADS), 0, s, a);
    } else {
        const dim3 grid((unsigned)((a.width + GS_CH - 1) / GS_CH), (unsigned)a.lanes.lanes);
        launch_pdl(mingru_wide_kernel, grid, dim3(GS_THREADS), 0, s, a);
    }
    MK_LAUNCH_CHECK();
}

}  // namespace mk
