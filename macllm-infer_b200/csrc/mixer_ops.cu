// See mixer_ops.h.
#include "mixer_ops.h"
#include "device_util.h"
#include "linear_state.h"
#include "recurrent_core.cuh"
#include <algorithm>

namespace mk {

namespace {

// ------------------------------------------------------------------------------------------------ residual update

constexpr int RU_THREADS = 256;

template <int VEC>
struct Pack {
    float v[VEC];
};
template <int VEC>
__device__ __forceinline__ Pack<VEC> load_pack(const float* p) {
    Pack<VEC> r;
    if constexpr (VEC == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int VEC>
__device__ __forceinline__ void store_pack(float* p, const Pack<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int VEC>
__device__ __forceinline__ Pack<VEC> share_pack(const Shares& s, int64_t row, int col) {
    Pack<VEC> r;
    if constexpr (VEC == 4) {
        const float4 x = s.at4(row, col);
        r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
    } else {
        r.v[0] = s.at(row, col);
    }
    return r;
}
template <int VEC>
__device__ __forceinline__ void put_pack(const RowImage& im, int64_t row, int col, const Pack<VEC>& r) {
    if constexpr (VEC == 4) im.put4(row, col, make_float4(r.v[0], r.v[1], r.v[2], r.v[3]));
    else im.put(row, col, r.v[0]);
}

__device__ __forceinline__ void zero_tail(const RowImage& im, int64_t row, int width) {
    for (int c = width + threadIdx.x; c < im.end(); c += blockDim.x) im.put(row, c, 0.f);
}

// VEC values of branch b of a row: the matmul's, the chosen experts' and the bias.
template <int VEC>
__device__ __forceinline__ Pack<VEC> branch_pack(const RowUpdateArgs& a, int b, int64_t row, int c) {
    Pack<VEC> y;
    if (a.add[b].p != nullptr) {
        y = share_pack<VEC>(a.add[b], row, c);
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) y.v[i] = 0.f;
    }
    for (int j = 0; j < a.routed_k; ++j) {
        const Pack<VEC> e = load_pack<VEC>(a.routed + (int64_t)a.routed_at[row * a.routed_k + j] * a.width + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y.v[i] += e.v[i];
    }
    if (a.add_bias != nullptr) {
        const Pack<VEC> e = load_pack<VEC>(a.add_bias + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y.v[i] += e.v[i];
    }
    return y;
}

// The updated row into `dst` (shared memory): x + coef * (branches + bias).  Normed branches are staged in `dst` / `other` first.
template <int VEC>
__device__ __forceinline__ void updated_row(const RowUpdateArgs& a, int64_t row, float* dst, float* other, float* red) {
    const int step = RU_THREADS * VEC;
    float inv[2] = {1.f, 1.f};
    const bool normed = a.n_add > 0 && a.add_w[0] != nullptr;
    if (normed) {
        for (int b = 0; b < a.n_add; ++b) {
            float* st = b == 0 ? dst : other;
            float ss = 0.f;
            for (int c = threadIdx.x * VEC; c < a.width; c += step) {
                const Pack<VEC> y = branch_pack<VEC>(a, b, row, c);
                store_pack<VEC>(st + c, y);
#pragma unroll
                for (int i = 0; i < VEC; ++i) ss = fmaf(y.v[i], y.v[i], ss);
            }
            ss = block_sum(ss, red);
            inv[b] = sqrtf(ss / (float)a.width + a.add_eps);
        }
    }
    // a thread reads and writes the same columns of the staging rows throughout, so no barrier is needed in between
    for (int c = threadIdx.x * VEC; c < a.width; c += step) {
        Pack<VEC> v;
        if (a.x != nullptr) v = load_pack<VEC>(a.x + row * a.width + c);
        else
#pragma unroll
            for (int i = 0; i < VEC; ++i) v.v[i] = 0.f;
        if (normed) {
            Pack<VEC> sum;
            const Pack<VEC> y0 = load_pack<VEC>(dst + c), w0 = load_pack<VEC>(a.add_w[0] + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) sum.v[i] = y0.v[i] / inv[0] * w0.v[i];
            if (a.n_add > 1) {
                const Pack<VEC> y1 = load_pack<VEC>(other + c), w1 = load_pack<VEC>(a.add_w[1] + c);
#pragma unroll
                for (int i = 0; i < VEC; ++i) sum.v[i] += y1.v[i] / inv[1] * w1.v[i];
            }
#pragma unroll
            for (int i = 0; i < VEC; ++i) v.v[i] = fmaf(a.add_coef, sum.v[i], v.v[i]);
        } else if (a.n_add > 0) {
            const Pack<VEC> y = branch_pack<VEC>(a, 0, row, c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) v.v[i] = fmaf(a.add_coef, y.v[i], v.v[i]);
        }
        store_pack<VEC>(dst + c, v);
    }
}

// Mean and root of (variance + eps) of a staged row, for the layer norm; root of (mean square + eps) for the RMS norm.
struct RowStats {
    float mean = 0.f, root = 1.f;
};
template <int VEC>
__device__ __forceinline__ RowStats row_stats(const float* x, int width, float eps, float* red, bool centred = true) {
    const int step = RU_THREADS * VEC;
    float s = 0.f;
    RowStats r;
    if (centred) {
        for (int c = threadIdx.x * VEC; c < width; c += step) {
            const Pack<VEC> v = load_pack<VEC>(x + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) s += v.v[i];
        }
        r.mean = block_sum(s, red) / (float)width;
    }
    s = 0.f;
    for (int c = threadIdx.x * VEC; c < width; c += step) {
        const Pack<VEC> v = load_pack<VEC>(x + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s = fmaf(v.v[i] - r.mean, v.v[i] - r.mean, s);
    }
    r.root = sqrtf(block_sum(s, red) / (float)width + eps);
    return r;
}

template <int VEC>
__device__ __forceinline__ Pack<VEC> norm_pack(const RowUpdateArgs& a, const RowStats& st, const Pack<VEC>& x, int c) {
    Pack<VEC> h;
    const Pack<VEC> w = load_pack<VEC>(a.norm_w + c);
    if (a.norm != NormKind::DynTanh) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) h.v[i] = (x.v[i] - st.mean) / st.root * w.v[i];
    } else {
        const Pack<VEC> b = load_pack<VEC>(a.norm_b + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) h.v[i] = fmaf(tanhf(a.alpha * x.v[i]), w.v[i], b.v[i]);
    }
    return h;
}

// Shared memory: the row, its neighbour (n_mix > 0), and a staging row for a second normed branch.
template <int VEC>
__global__ void __launch_bounds__(RU_THREADS) row_update_kernel(RowUpdateArgs a) {
    extern __shared__ __align__(16) float ru_smem[];
    __shared__ float red[32];
    float* cur = ru_smem;
    float* prv = cur + (a.n_mix > 0 ? a.width : 0);
    float* other = prv + a.width;
    pdl_trigger();
    pdl_wait();
    const int64_t r = blockIdx.x;
    const int64_t row = a.row_index ? a.row_index[r] : r;
    const int step = RU_THREADS * VEC;
    updated_row<VEC>(a, row, cur, other, red);
    if (a.x_out != nullptr)
        for (int c = threadIdx.x * VEC; c < a.width; c += step) store_pack<VEC>(a.x_out + row * a.width + c, load_pack<VEC>(cur + c));
    if (a.raw.any()) {
        for (int c = threadIdx.x * VEC; c < a.width; c += step) put_pack<VEC>(a.raw, r, c, load_pack<VEC>(cur + c));
        zero_tail(a.raw, r, a.width);
    }
    if (a.norm == NormKind::None) return;
    // a thread has written the columns of `cur` that it reads itself; block_sum's barriers are all the sums need
    RowStats st, st_prev;
    const bool stats = a.norm != NormKind::DynTanh, centred = a.norm == NormKind::Layer;
    if (stats) st = row_stats<VEC>(cur, a.width, a.norm_eps, red, centred);
    if (a.n_mix == 0) {
        for (int c = threadIdx.x * VEC; c < a.width; c += step) put_pack<VEC>(a.normed, r, c, norm_pack<VEC>(a, st, load_pack<VEC>(cur + c), c));
        zero_tail(a.normed, r, a.width);
        return;
    }
    const int lane = a.token_lane[row];
    const StateLane sl = a.lanes.at(lane);
    const int first = sl.first, last = sl.first + sl.n - 1;
    const bool inside = row > first;
    if (inside) {
        updated_row<VEC>(a, row - 1, prv, other, red);
        if (stats) st_prev = row_stats<VEC>(prv, a.width, a.norm_eps, red, centred);
    }
    for (int c = threadIdx.x * VEC; c < a.width; c += step) {
        const Pack<VEC> h = norm_pack<VEC>(a, st, load_pack<VEC>(cur + c), c);
        Pack<VEC> p;
        if (inside) p = norm_pack<VEC>(a, st_prev, load_pack<VEC>(prv + c), c);
        else if (sl.in >= 0) p = load_pack<VEC>(a.kept + (int64_t)sl.in * a.width + c);
        else
#pragma unroll
            for (int i = 0; i < VEC; ++i) p.v[i] = 0.f;
        for (int m = 0; m < a.n_mix; ++m) {
            const Pack<VEC> mu = load_pack<VEC>(a.mu + (int64_t)m * a.width + c);
            Pack<VEC> o;
#pragma unroll
            for (int i = 0; i < VEC; ++i) o.v[i] = fmaf(p.v[i] - h.v[i], mu.v[i], h.v[i]);
            put_pack<VEC>(a.mixes, (int64_t)m * a.rows + r, c, o);
        }
        if (row == last) store_pack<VEC>(a.kept + (int64_t)sl.out * a.width + c, h);
    }
    for (int m = 0; m < a.n_mix; ++m) zero_tail(a.mixes, (int64_t)m * a.rows + r, a.width);
}

// Rows of a short convolution: a CTA takes ROWS consecutive rows and the taps - 1 before them (of the first one's lane), updates them
// all into shared memory behind one barrier for their sums of squares, and then walks its columns down the rows with the last taps - 1
// normed rows in registers (TAPS > 0) or in the staged rows (any number of taps).  A thread reads the columns it has staged itself.
template <int VEC, int ROWS, int TAPS>
__global__ void __launch_bounds__(RU_THREADS) conv_update_kernel(RowUpdateArgs a) {
    extern __shared__ __align__(16) float cu_smem[];   // [ROWS + taps - 1][width], then [ROWS + taps - 1] sums per warp and inverse roots
    constexpr int BATCH = ROWS >= 4 ? 4 : ROWS;
    constexpr int WARPS = RU_THREADS / 32;
    const int taps = TAPS > 0 ? TAPS : a.taps, hist = taps - 1, staged = ROWS + hist, W = a.width;
    float* red = cu_smem + (int64_t)staged * W;
    float* inv = red + staged * WARPS;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, step = RU_THREADS * VEC;
    pdl_trigger();
    pdl_wait();
    const int r0 = blockIdx.x * ROWS, r1 = min(a.rows, r0 + ROWS);
    StateLane sl = a.lanes.at(a.token_lane[r0]);
    const int lo = max(max(0, sl.first), r0 - hist), n = r1 - lo;
    for (int i0 = 0; i0 < n; i0 += BATCH) {
        float ss[BATCH];
#pragma unroll
        for (int u = 0; u < BATCH; ++u) ss[u] = 0.f;
        for (int c = threadIdx.x * VEC; c < W; c += step) {
            Pack<VEC> v[BATCH];
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                if (i0 + u >= n) continue;
                v[u] = load_pack<VEC>(a.x + (int64_t)(lo + i0 + u) * W + c);
            }
            if (a.n_add > 0) {
#pragma unroll
                for (int u = 0; u < BATCH; ++u) {
                    if (i0 + u >= n) continue;
                    const Pack<VEC> y = branch_pack<VEC>(a, 0, lo + i0 + u, c);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) v[u].v[i] = fmaf(a.add_coef, y.v[i], v[u].v[i]);
                }
            }
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                if (i0 + u >= n) continue;
                const int row = lo + i0 + u;
                if (row >= r0 && a.x_out != nullptr) store_pack<VEC>(a.x_out + (int64_t)row * W + c, v[u]);
                store_pack<VEC>(cu_smem + (int64_t)(i0 + u) * W + c, v[u]);
#pragma unroll
                for (int i = 0; i < VEC; ++i) ss[u] = fmaf(v[u].v[i], v[u].v[i], ss[u]);
            }
        }
#pragma unroll
        for (int u = 0; u < BATCH; ++u) {
            const float s = warp_sum(ss[u]);
            if (lane == 0 && i0 + u < n) red[(i0 + u) * WARPS + warp] = s;
        }
    }
    __syncthreads();
    // every thread needs every row's root: the first threads add one up each
    for (int i = threadIdx.x; i < n; i += RU_THREADS) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) s += red[i * WARPS + w];
        inv[i] = 1.0f / sqrtf(s / (float)W + a.norm_eps);
    }
    __syncthreads();
    const StateLane first_lane = sl;
    for (int c = threadIdx.x * VEC; c < W; c += step) {
        const Pack<VEC> w = load_pack<VEC>(a.norm_w + c);
        sl = first_lane;
        auto normed = [&](int row) {  // h of a row of the lane, or of one before this tick
            Pack<VEC> h;
            if (row >= sl.first) {
                h = load_pack<VEC>(cu_smem + (int64_t)(row - lo) * W + c);
                const float d = inv[row - lo];
#pragma unroll
                for (int i = 0; i < VEC; ++i) h.v[i] = h.v[i] * d * w.v[i];
            } else if (sl.in >= 0) {
                h = load_pack<VEC>(a.kept + ((int64_t)sl.in * hist + hist + row - sl.first) * W + c);
            } else {
#pragma unroll
                for (int i = 0; i < VEC; ++i) h.v[i] = 0.f;
            }
            return h;
        };
        if constexpr (TAPS > 0) {
            Pack<VEC> k[TAPS], win[TAPS];  // win[j]: h of the row TAPS - 1 - j before
#pragma unroll
            for (int j = 0; j < TAPS; ++j) k[j] = load_pack<VEC>(a.conv + (int64_t)j * W + c);
#pragma unroll
            for (int j = 0; j < hist; ++j) win[j + 1] = normed(r0 - hist + j);
            for (int r = r0; r < r1; ++r) {
                if (r >= sl.first + sl.n) {
                    sl = a.lanes.at(a.token_lane[r]);
#pragma unroll
                    for (int j = 0; j < hist; ++j) win[j + 1] = normed(r - hist + j);
                }
#pragma unroll
                for (int j = 0; j < hist; ++j) win[j] = win[j + 1];
                win[hist] = normed(r);
                Pack<VEC> sum = win[hist];
#pragma unroll
                for (int j = 0; j < TAPS; ++j)
#pragma unroll
                    for (int i = 0; i < VEC; ++i) sum.v[i] = fmaf(k[j].v[i], win[j].v[i], sum.v[i]);
                put_pack<VEC>(a.normed, r, c, sum);
                if (r == sl.first + sl.n - 1)
#pragma unroll
                    for (int t = 0; t < hist; ++t) store_pack<VEC>(a.kept + ((int64_t)sl.out * hist + t) * W + c, win[t + 1]);
            }
        } else {
            for (int r = r0; r < r1; ++r) {
                if (r >= sl.first + sl.n) sl = a.lanes.at(a.token_lane[r]);
                Pack<VEC> sum = normed(r);
                for (int j = 0; j < taps; ++j) {
                    const Pack<VEC> k = load_pack<VEC>(a.conv + (int64_t)j * W + c), h = normed(r - hist + j);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) sum.v[i] = fmaf(k.v[i], h.v[i], sum.v[i]);
                }
                put_pack<VEC>(a.normed, r, c, sum);
                if (r == sl.first + sl.n - 1)
                    for (int t = 0; t < hist; ++t) store_pack<VEC>(a.kept + ((int64_t)sl.out * hist + t) * W + c, normed(r - hist + 1 + t));
            }
        }
    }
    for (int r = r0; r < r1; ++r) zero_tail(a.normed, r, W);
}

template <int VEC, int ROWS, int TAPS>
void launch_conv_taps(const RowUpdateArgs& a, cudaStream_t s) {
    const size_t staged = (size_t)ROWS + a.taps - 1, smem = (staged * a.width + staged * (RU_THREADS / 32 + 1)) * 4;
    if (smem > (size_t)220 * 1024) throw std::runtime_error("launch_row_update: the model is too wide for its short convolution");
    ensure_dynamic_smem(reinterpret_cast<const void*>(&conv_update_kernel<VEC, ROWS, TAPS>), smem);
    launch_pdl(conv_update_kernel<VEC, ROWS, TAPS>, dim3((unsigned)((a.rows + ROWS - 1) / ROWS)), dim3(RU_THREADS), smem, s, a);
}

template <int VEC, int ROWS>
void launch_conv_rows(const RowUpdateArgs& a, cudaStream_t s) {
    if (a.taps == 4) launch_conv_taps<VEC, ROWS, 4>(a, s);
    else launch_conv_taps<VEC, ROWS, 0>(a, s);
}

// ------------------------------------------------------------------------------------------------ WKV decay

constexpr int WD_COLS = 128;       // channels (threads) of a CTA
constexpr int WD_STAGE_RANK = 256; // up to this rank the CTA's slice of w2 is staged, on its way before the predecessor is done

template <int ROWS>
__global__ void __launch_bounds__(WD_COLS) wkv_decay_kernel(Shares low, int low_col, int rows, int rank, int channels,
                                                            const float* __restrict__ w2t, const float* __restrict__ w0, float* decay) {
    extern __shared__ __align__(16) float wd_smem[];
    float* z = wd_smem;                // [rank][ROWS]
    float* ws = z + rank * ROWS;       // [rank][WD_COLS]
    const int r0 = blockIdx.y * ROWS, c = blockIdx.x * WD_COLS + threadIdx.x;
    const bool staged = rank <= WD_STAGE_RANK, live = c < channels;
    pdl_trigger();
    if (staged && live)
        for (int j = 0; j < rank; ++j)
            asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(ws + j * WD_COLS + threadIdx.x)),
                         "l"(w2t + (int64_t)j * channels + c)
                         : "memory");
    asm volatile("cp.async.commit_group;" ::: "memory");
    pdl_wait();
    for (int i = threadIdx.x; i < rank * ROWS; i += WD_COLS) {
        const int r = i / rank, j = i - r * rank;
        z[j * ROWS + r] = r0 + r < rows ? tanhf(low.at(r0 + r, low_col + j)) : 0.f;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (!live) return;
    float acc[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) acc[r] = 0.f;
#pragma unroll 4
    for (int j = 0; j < rank; ++j) {
        const float w = staged ? ws[j * WD_COLS + threadIdx.x] : w2t[(int64_t)j * channels + c];
#pragma unroll
        for (int r = 0; r < ROWS; r += 4) {
            const float4 v = *reinterpret_cast<const float4*>(z + j * ROWS + r);
            acc[r] = fmaf(v.x, w, acc[r]);
            acc[r + 1] = fmaf(v.y, w, acc[r + 1]);
            acc[r + 2] = fmaf(v.z, w, acc[r + 2]);
            acc[r + 3] = fmaf(v.w, w, acc[r + 3]);
        }
    }
    const float b = w0[c];
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
        if (r0 + r < rows) decay[(int64_t)(r0 + r) * channels + c] = expf(-expf(acc[r] + b));
}

template <int ROWS>
void launch_decay_rows(const Shares& low, int low_col, int rows, int rank, int channels, const float* w2t, const float* w0, float* decay, cudaStream_t s) {
    const size_t smem = ((size_t)rank * ROWS + (rank <= WD_STAGE_RANK ? (size_t)rank * WD_COLS : 0)) * 4;
    if (smem > (size_t)220 * 1024) throw std::runtime_error("launch_wkv_decay: the low rank is too large");
    ensure_dynamic_smem(reinterpret_cast<const void*>(&wkv_decay_kernel<ROWS>), smem);
    const dim3 grid((unsigned)((channels + WD_COLS - 1) / WD_COLS), (unsigned)((rows + ROWS - 1) / ROWS));
    launch_pdl(wkv_decay_kernel<ROWS>, grid, dim3(WD_COLS), smem, s, low, low_col, rows, rank, channels, w2t, w0, decay);
    MK_LAUNCH_CHECK();
}

// ------------------------------------------------------------------------------------------------ channel gates of the delta rule

// A CTA takes ROWS rows and whole heads of up to CG_COLS channels together, a channel per thread.
constexpr int CG_COLS = 256;

template <int ROWS>
__global__ void __launch_bounds__(CG_COLS) channel_gates_kernel(ChannelGatesArgs a, int tile_heads) {
    extern __shared__ __align__(16) float cg_smem[];
    const int cols = tile_heads * a.dim, channels = a.heads * a.dim;
    float* z = cg_smem;                       // [rank][ROWS]
    float* ks = z + a.rank * ROWS;            // [ROWS][cols]
    float* inv = ks + ROWS * cols;            // [ROWS][tile_heads]
    const StateLane sl = a.lanes.at(blockIdx.z);
    const int r0 = sl.first + blockIdx.y * ROWS, end = sl.first + sl.n, c = blockIdx.x * cols + threadIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    if (r0 >= end) return;
    const bool live = (int)threadIdx.x < cols && c < channels;
    pdl_trigger();
    pdl_wait();
    for (int i = threadIdx.x; i < a.rank * ROWS; i += blockDim.x) {
        const int r = i / a.rank, j = i - r * a.rank;
        z[j * ROWS + r] = r0 + r < end ? tanhf(a.y.at(r0 + r, a.low_col + j)) : 0.f;
    }
    float k[ROWS], gate[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const bool there = live && r0 + r < end;
        k[r] = there ? a.y.at(r0 + r, a.k_col + c) : 0.f;
        gate[r] = there ? a.y.at(r0 + r, a.a_col + c) : 0.f;
        if ((int)threadIdx.x < cols) ks[r * cols + threadIdx.x] = k[r];
    }
    __syncthreads();
    for (int i = warp; i < ROWS * tile_heads; i += warps) {
        const float* row = ks + i / tile_heads * cols + i % tile_heads * a.dim;
        float ss = 0.f;
        for (int d = lane; d < a.dim; d += 32) ss = fmaf(row[d], row[d], ss);
        ss = warp_sum(ss);
        if (lane == 0) inv[i] = 1.0f / (ss + 1e-6f);
    }
    float acc[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) acc[r] = 0.f;
    if (live) {
#pragma unroll 8
        for (int j = 0; j < a.rank; ++j) {
            const float w = a.w2t[(int64_t)j * channels + c];
#pragma unroll
            for (int r = 0; r < ROWS; r += 4) {
                const float4 v = *reinterpret_cast<const float4*>(z + j * ROWS + r);
                acc[r] = fmaf(v.x, w, acc[r]);
                acc[r + 1] = fmaf(v.y, w, acc[r + 1]);
                acc[r + 2] = fmaf(v.z, w, acc[r + 2]);
                acc[r + 3] = fmaf(v.w, w, acc[r + 3]);
            }
        }
    }
    __syncthreads();
    if (!live) return;
    const float w0 = a.w0[c], bias = a.a_bias[c];
    const int head = threadIdx.x / a.dim;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        if (r0 + r >= end) break;
        const int64_t at = (int64_t)(r0 + r) * channels + c;
        a.decay[at] = channel_decay_f(acc[r] + w0);
        a.removal[at] = sigmoid_f(gate[r] + bias) * k[r] * inv[r * tile_heads + head];
    }
}

template <int ROWS>
void launch_channel_rows(const ChannelGatesArgs& a, cudaStream_t s) {
    const int tile_heads = std::min(a.heads, std::max(1, 128 / a.dim)), cols = tile_heads * a.dim;
    const size_t smem = ((size_t)a.rank * ROWS + (size_t)ROWS * (cols + tile_heads)) * 4;
    if (smem > (size_t)220 * 1024) throw std::runtime_error("launch_channel_gates: the low rank is too large");
    ensure_dynamic_smem(reinterpret_cast<const void*>(&channel_gates_kernel<ROWS>), smem);
    const dim3 grid((unsigned)((a.heads + tile_heads - 1) / tile_heads), (unsigned)((a.longest + ROWS - 1) / ROWS), (unsigned)a.lanes.lanes);
    launch_pdl(channel_gates_kernel<ROWS>, grid, dim3((unsigned)((cols + 31) / 32 * 32)), smem, s, a, tile_heads);
    MK_LAUNCH_CHECK();
}

// ------------------------------------------------------------------------------------------------ delta-rule inputs

constexpr int DP_WARPS = 4;
constexpr int DP_MAX_DIM = 256;
constexpr int DP_ROWS = 4;   // rows a warp walks on wide ticks: their windows overlap and stay in L1

// VEC neighbouring channels of the raw projection at row i of the lane (negative: before this tick).
template <int VEC>
__device__ __forceinline__ Pack<VEC> raw_pack(const DeltaPrepArgs& a, const StateLane& sl, int i, int ch, int y_col, int channels) {
    if (i >= 0) return share_pack<VEC>(a.y, sl.first + i, y_col);
    if (sl.in >= 0) return load_pack<VEC>(a.tail + ((int64_t)sl.in * (a.taps - 1) + (a.taps - 1 + i)) * channels + ch);
    Pack<VEC> z;
#pragma unroll
    for (int e = 0; e < VEC; ++e) z.v[e] = 0.f;
    return z;
}

// A warp takes one head of q, k or v and a run of consecutive packed rows; a lane takes VEC neighbouring channels of every 32 * VEC.
template <int VEC>
__global__ void __launch_bounds__(DP_WARPS * 32) delta_prep_kernel(DeltaPrepArgs a, int run) {
    constexpr int NE = DP_MAX_DIM / 32 / VEC;
    const int kw = a.kv_heads * a.dim, vw = a.heads * a.vdim, channels = 2 * kw + vw;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int u = blockIdx.y * DP_WARPS + warp, units = 2 * a.kv_heads + a.heads;
    pdl_trigger();
    pdl_wait();
    const int r0 = blockIdx.x * run, r1 = min(a.rows, r0 + run);
    if (blockIdx.y == 0)
        for (int i = threadIdx.x; i < (r1 - r0) * a.heads; i += DP_WARPS * 32) {
            const int row = r0 + i / a.heads, h = i % a.heads;
            a.beta[(int64_t)row * a.heads + h] = sigmoid_f(a.y.at(row, a.b_col + h));
            a.decay[(int64_t)row * a.heads + h] = recurrent::gated_delta_decay(a.y.at(row, a.a_col + h), a.dt_bias[h], a.log_decay[h]);
        }
    if (u >= units) return;
    const int kind = u < a.kv_heads ? 0 : (u < 2 * a.kv_heads ? 1 : 2);
    const int head = kind == 0 ? u : (kind == 1 ? u - a.kv_heads : u - 2 * a.kv_heads);
    const int dim = kind == 2 ? a.vdim : a.dim;
    const int ch0 = (kind == 0 ? 0 : (kind == 1 ? kw : 2 * kw)) + head * dim;
    const int y0 = (kind == 0 ? a.q_col : (kind == 1 ? a.k_col : a.v_col)) + head * dim;
    float* out = (kind == 0 ? a.q : (kind == 1 ? a.k : a.v)) + head * dim;
    const int ldo = kind == 2 ? vw : kw;
    const int hist = a.taps - 1;
    int seq = -1;
    StateLane sl{};
    for (int row = r0; row < r1; ++row) {
        if (seq < 0 || row >= sl.first + sl.n) {
            seq = a.token_lane[row];
            sl = a.lanes.at(seq);
        }
        const int i = row - sl.first;
        Pack<VEC> val[NE];
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < NE; ++e) {
            const int c = (e * 32 + lane) * VEC;
            if (c >= dim) continue;
            Pack<VEC> sum;
#pragma unroll
            for (int x = 0; x < VEC; ++x) sum.v[x] = 0.f;
#pragma unroll 4
            for (int j = 0; j < a.taps; ++j) {
                const Pack<VEC> w = load_pack<VEC>(a.conv + (int64_t)j * channels + ch0 + c);
                const Pack<VEC> r = raw_pack<VEC>(a, sl, i - hist + j, ch0 + c, y0 + c, channels);
#pragma unroll
                for (int x = 0; x < VEC; ++x) sum.v[x] = fmaf(w.v[x], r.v[x], sum.v[x]);
            }
#pragma unroll
            for (int x = 0; x < VEC; ++x) {
                val[e].v[x] = silu_f(sum.v[x]);
                ss = fmaf(val[e].v[x], val[e].v[x], ss);
            }
        }
        float f = 1.f;
        if (kind != 2) {
            ss = warp_sum(ss);
            f = 1.0f / sqrtf(ss + 1e-6f);
            if (kind == 0) f *= rsqrtf((float)a.dim);
        }
#pragma unroll
        for (int e = 0; e < NE; ++e) {
            const int c = (e * 32 + lane) * VEC;
            if (c >= dim) continue;
#pragma unroll
            for (int x = 0; x < VEC; ++x) val[e].v[x] *= f;
            store_pack<VEC>(out + (int64_t)row * ldo + c, val[e]);
        }
        if (i == sl.n - 1)  // the raw rows the next forward starts from
            for (int t = 0; t < hist; ++t)
                for (int c = lane * VEC; c < dim; c += 32 * VEC)
                    store_pack<VEC>(a.tail + ((int64_t)sl.out * hist + t) * channels + ch0 + c,
                                    raw_pack<VEC>(a, sl, i - hist + 1 + t, ch0 + c, y0 + c, channels));
    }
}

// ------------------------------------------------------------------------------------------------ gates

__global__ void __launch_bounds__(256) head_gate_kernel(const float* attn, int heads, int row_width, int vdim, Shares gate, int gate_col, RowImage out,
                                                        const int32_t* rows, OutputGate kind, int vec_gate, float scale) {
    extern __shared__ float hg_gate[];
    pdl_trigger();
    pdl_wait();
    const int64_t row = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
    for (int h = threadIdx.x; h < heads; h += blockDim.x) hg_gate[h] = scale * (kind == OutputGate::Head ? sigmoid_f(gate.at(row, gate_col + h)) : 1.f);
    __syncthreads();
    const float* src = attn + row * heads * row_width;
    if ((vdim & 3) == 0) {  // out.end() is a multiple of 64, a head's row of 4
        for (int c = threadIdx.x * 4; c < out.end(); c += blockDim.x * 4) {
            const int h = c / vdim;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (h < heads) {
                v = *reinterpret_cast<const float4*>(src + h * row_width + (c - h * vdim));
                if (kind == OutputGate::Value) {
                    float4 g;
                    if (vec_gate) g = gate.at4(row, gate_col + c);
                    else g = make_float4(gate.at(row, gate_col + c), gate.at(row, gate_col + c + 1), gate.at(row, gate_col + c + 2), gate.at(row, gate_col + c + 3));
                    v = make_float4(scale * v.x * sigmoid_f(g.x), scale * v.y * sigmoid_f(g.y), scale * v.z * sigmoid_f(g.z), scale * v.w * sigmoid_f(g.w));
                } else {
                    const float g = hg_gate[h];
                    v = make_float4(v.x * g, v.y * g, v.z * g, v.w * g);
                }
            }
            out.put4(row, c, v);
        }
        return;
    }
    for (int c = threadIdx.x; c < out.end(); c += blockDim.x) {
        const int h = c / vdim;
        float v = 0.f;
        if (h < heads) v = src[h * row_width + (c - h * vdim)] * (kind == OutputGate::Value ? scale * sigmoid_f(gate.at(row, gate_col + c)) : hg_gate[h]);
        out.put(row, c, v);
    }
}

__global__ void __launch_bounds__(128) side_gate_kernel(Shares z, int dim, const uint32_t* ids, const void* table, int table_f32, int64_t table_ld,
                                                        int slice, RowImage out) {
    pdl_trigger();
    pdl_wait();
    const int64_t row = blockIdx.x;
    const int64_t at = (int64_t)ids[row] * table_ld + slice;
    for (int c = threadIdx.x; c < out.end(); c += blockDim.x) {
        float v = 0.f;
        if (c < dim) {
            const float e = table_f32 ? static_cast<const float*>(table)[at + c] : __bfloat162float(static_cast<const __nv_bfloat16*>(table)[at + c]);
            v = gelu_tanh_f(z.at(row, c)) * e;
        }
        out.put(row, c, v);
    }
}

__global__ void __launch_bounds__(256) gated_act_kernel(Shares gu, int ff, RowImage out, GatedAct act) {
    pdl_trigger();
    pdl_wait();
    const int64_t row = blockIdx.x;
    const float pre = act.pre != nullptr ? act.pre[row] : 1.f, post = act.post != nullptr ? act.post[row] : 1.f;
    for (int c = threadIdx.x; c < out.end(); c += blockDim.x) {
        float v = 0.f;
        if (c < ff) {
            const float g = gu.at(row, 2 * c), u = gu.at(row, 2 * c + 1);
            v = act.kind == GatedAct::Clamped ? clamped_gate_f(pre * g, pre * u, act.limit) * post : (act.kind == GatedAct::Silu ? silu_f(g) : gelu_tanh_f(g)) * u;
        }
        out.put(row, c, v);
    }
}

// ------------------------------------------------------------------------------------------------ embedding with positions

// Shared memory: the row.
__global__ void __launch_bounds__(RU_THREADS) embed_norm_kernel(EmbedNormArgs a) {
    extern __shared__ __align__(16) float en_row[];
    __shared__ float red[32];
    pdl_trigger();
    pdl_wait();
    const int64_t row = blockIdx.x, at = (int64_t)a.ids[row] * a.width;
    const double pos = (double)a.positions[row];
    constexpr double kTwoPi = 6.283185307179586476925;
    for (int i = threadIdx.x; 2 * i < a.width; i += RU_THREADS) {
        double angle = pos * a.freq[i];
        angle -= rint(angle / kTwoPi) * kTwoPi;
        float sn, cs;
        sincosf((float)angle, &sn, &cs);
        for (int j = 0; j < 2 && 2 * i + j < a.width; ++j) {
            const int c = 2 * i + j;
            const float e = a.table_f32 ? static_cast<const float*>(a.table)[at + c] : __bfloat162float(static_cast<const __nv_bfloat16*>(a.table)[at + c]);
            en_row[c] = e + (j == 0 ? sn : cs);
        }
    }
    __syncthreads();
    const RowStats st = row_stats<1>(en_row, a.width, a.eps, red);
    for (int c = threadIdx.x; c < a.width; c += RU_THREADS) {
        const float v = (en_row[c] - st.mean) / st.root * a.norm_w[c];
        a.x[row * a.width + c] = v;
        if (a.image.any()) a.image.put(row, c, v);
    }
    if (a.image.any()) zero_tail(a.image, row, a.width);
}

// ------------------------------------------------------------------------------------------------ latents, polynomial activation

constexpr int LP_THREADS = 256;

// Three block sums behind one barrier.
__device__ __forceinline__ float3 block_sum3(float3 v, float (*red)[3]) {
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    v.x = warp_sum(v.x);
    v.y = warp_sum(v.y);
    v.z = warp_sum(v.z);
    if (lane == 0) {
        red[w][0] = v.x;
        red[w][1] = v.y;
        red[w][2] = v.z;
    }
    __syncthreads();
    float3 r = make_float3(0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < LP_THREADS / 32; ++i) {
        r.x += red[i][0];
        r.y += red[i][1];
        r.z += red[i][2];
    }
    return r;
}

template <int VEC>
__device__ __forceinline__ void poly_row(const LatentPrepArgs& a, int64_t row, float* z, float (*red)[3]) {
    const int step = LP_THREADS * VEC;
    float3 ss = make_float3(0.f, 0.f, 0.f);
    for (int c = threadIdx.x * VEC; c < a.ff; c += step) {
        Pack<VEC> v = share_pack<VEC>(a.y, row, a.ff_col + c);
        const Pack<VEC> b = load_pack<VEC>(a.ff_bias + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            v.v[i] += b.v[i];
            const float z1 = v.v[i], z2 = z1 * z1, z3 = z2 * z1;
            ss.x = fmaf(z1, z1, ss.x);
            ss.y = fmaf(z2, z2, ss.y);
            ss.z = fmaf(z3, z3, ss.z);
        }
        store_pack<VEC>(z + c, v);
    }
    ss = block_sum3(ss, red);
    const float n = (float)a.ff;
    const float k1 = a.poly[0] / sqrtf(ss.x / n + a.eps), k2 = a.poly[1] / sqrtf(ss.y / n + a.eps), k3 = a.poly[2] / sqrtf(ss.z / n + a.eps), k0 = a.poly[3];
    for (int c = threadIdx.x * VEC; c < a.ff; c += step) {
        Pack<VEC> v = load_pack<VEC>(z + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v.v[i] = fmaf(fmaf(fmaf(k3, v.v[i], k2), v.v[i], k1), v.v[i], k0);
        put_pack<VEC>(a.ff_image, row, c, v);
    }
    zero_tail(a.ff_image, row, a.ff);
}

// Shared memory: max(ff, q_rank + kv_rank + rot_width) floats.
template <int VEC>
__global__ void __launch_bounds__(LP_THREADS) latent_prep_kernel(LatentPrepArgs a) {
    extern __shared__ __align__(16) float lp_row[];
    __shared__ float red[LP_THREADS / 32][3];
    pdl_trigger();
    pdl_wait();
    const int64_t row = blockIdx.x;
    if (a.q_rank == 0 || blockIdx.y == 1) {
        poly_row<VEC>(a, row, lp_row, red);
        return;
    }
    float *kv = lp_row + a.q_rank, *rot = kv + a.kv_rank;
    const int64_t at = a.slots[row] * a.kv_width, turn0 = a.rot_dims > 0 ? (int64_t)a.positions[row] * (a.rot_dims / 2) : 0;
    float3 ss = make_float3(0.f, 0.f, 0.f);
    // a latent's raw values into shared memory; returns the thread's sum of squares
    auto stage = [&](float* dst, int n, int col) {
        float s = 0.f;
        if (a.lat_vec) {
            for (int c = threadIdx.x * 4; c < n; c += LP_THREADS * 4) {
                const float4 v = a.y.at4(row, col + c);
                *reinterpret_cast<float4*>(dst + c) = v;
                s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
            }
        } else {
            for (int c = threadIdx.x; c < n; c += LP_THREADS) {
                const float v = a.y.at(row, col + c);
                dst[c] = v;
                s = fmaf(v, v, s);
            }
        }
        return s;
    };
    ss.x = stage(lp_row, a.q_rank, a.q_col);
    ss.y = stage(kv, a.kv_rank, a.kv_col);
    for (int c = threadIdx.x; c < a.rot_width; c += LP_THREADS) rot[c] = a.y.at(row, a.rot_col + c);
    ss = block_sum3(ss, red);
    const float rq = sqrtf(ss.x / (float)a.q_rank + a.eps), rk = sqrtf(ss.y / (float)a.kv_rank + a.eps);
    if (a.lat_vec) {
        for (int c = threadIdx.x * 4; c < a.q_rank; c += LP_THREADS * 4) {
            const float4 v = *reinterpret_cast<const float4*>(lp_row + c), w = *reinterpret_cast<const float4*>(a.q_norm + c);
            a.q_image.put4(row, c, make_float4(v.x / rq * w.x, v.y / rq * w.y, v.z / rq * w.z, v.w / rq * w.w));
        }
    } else {
        for (int c = threadIdx.x; c < a.q_rank; c += LP_THREADS) a.q_image.put(row, c, lp_row[c] / rq * a.q_norm[c]);
    }
    zero_tail(a.q_image, row, a.q_rank);
    auto value = [&](int c) {  // column c of the page row
        if (c < a.kv_rank) return kv[c] / rk * a.kv_norm[c];
        const int i = c - a.rot0;
        if (i < 0 || i >= a.rot_width) return 0.f;
        if (i >= a.rot_dims) return rot[i];
        const float cs = a.cos_t[turn0 + (i >> 1)], sn = a.sin_t[turn0 + (i >> 1)];
        return (i & 1) == 0 ? rot[i] * cs - rot[i ^ 1] * sn : rot[i] * cs + rot[i ^ 1] * sn;
    };
    for (int c = threadIdx.x * 2; c < a.kv_width; c += LP_THREADS * 2) {  // a row is a multiple of 64 wide
        const float x = value(c), y = value(c + 1);
        if (a.pool_f16) *reinterpret_cast<__half2*>(static_cast<__half*>(a.pool) + at + c) = __floats2half2_rn(x, y);
        else *reinterpret_cast<float2*>(static_cast<float*>(a.pool) + at + c) = make_float2(x, y);
    }
}

// The latents of wide ticks, a warp per row: in whole packs of a finished matmul, read twice (the second time out of the cache).
__global__ void __launch_bounds__(LP_THREADS) latent_rows_kernel(LatentPrepArgs a) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const int64_t row = (int64_t)blockIdx.x * (LP_THREADS / 32) + (threadIdx.x >> 5);
    if (row >= a.rows) return;
    const float* y = a.y.p + row * a.y.ld;
    const int64_t at = a.slots[row] * a.kv_width, turn0 = a.rot_dims > 0 ? (int64_t)a.positions[row] * (a.rot_dims / 2) : 0;
    auto squares = [&](int n, int col) {
        float s = 0.f;
#pragma unroll 8
        for (int c = lane * 4; c < n; c += 128) {
            const float4 v = *reinterpret_cast<const float4*>(y + col + c);
            s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
        }
        return s;
    };
    float sq = squares(a.q_rank, a.q_col), sk = squares(a.kv_rank, a.kv_col);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    const float rq = sqrtf(sq / (float)a.q_rank + a.eps), rk = sqrtf(sk / (float)a.kv_rank + a.eps);
#pragma unroll 4
    for (int c = lane * 4; c < a.q_image.end(); c += 128) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < a.q_rank) {
            const float4 x = *reinterpret_cast<const float4*>(y + a.q_col + c), w = *reinterpret_cast<const float4*>(a.q_norm + c);
            v = make_float4(x.x / rq * w.x, x.y / rq * w.y, x.z / rq * w.z, x.w / rq * w.w);
        }
        a.q_image.put4(row, c, v);
    }
    auto rotated = [&](int i) {
        const float v = y[a.rot_col + i];
        if (i >= a.rot_dims) return v;
        const float other = y[a.rot_col + (i ^ 1)], cs = a.cos_t[turn0 + (i >> 1)], sn = a.sin_t[turn0 + (i >> 1)];
        return (i & 1) == 0 ? v * cs - other * sn : v * cs + other * sn;
    };
#pragma unroll 4
    for (int c = lane * 4; c < a.kv_width; c += 128) {
        float v[4] = {};
        if (c < a.kv_rank) {
            const float4 x = *reinterpret_cast<const float4*>(y + a.kv_col + c), w = *reinterpret_cast<const float4*>(a.kv_norm + c);
            v[0] = x.x / rk * w.x; v[1] = x.y / rk * w.y; v[2] = x.z / rk * w.z; v[3] = x.w / rk * w.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = c + e - a.rot0;
                if (i >= 0 && i < a.rot_width) v[e] = rotated(i);
            }
        }
        if (a.pool_f16) {
            const __half2 lo = __floats2half2_rn(v[0], v[1]), hi = __floats2half2_rn(v[2], v[3]);
            *reinterpret_cast<uint2*>(static_cast<__half*>(a.pool) + at + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        } else {
            *reinterpret_cast<float4*>(static_cast<float*>(a.pool) + at + c) = make_float4(v[0], v[1], v[2], v[3]);
        }
    }
}

// ------------------------------------------------------------------------------------------------ f32 matmul

constexpr int FM_TILE = 64, FM_K = 16;

// 64 x 64 outputs per CTA, 4 x 4 per thread.
__global__ void __launch_bounds__(256) f32_matmul_kernel(const float* __restrict__ w, int64_t rows, int cols, const float* __restrict__ x, int T, float* y,
                                                         int ldy, float scale, float softcap, int n_groups, int group_tiles, int4 end_lo, int4 end_hi,
                                                         MatmulScatter to, const int32_t* __restrict__ offsets, int64_t matrix_rows) {
    __shared__ float ws[FM_K][FM_TILE + 4], xs[FM_K][FM_TILE + 4];
    pdl_trigger();
    pdl_wait();
    const int64_t n0 = (int64_t)blockIdx.x * FM_TILE;
    const int t0 = blockIdx.y * FM_TILE;
    if (offsets != nullptr) {  // rows grouped by expert: matrix blockIdx.z
        const int e = blockIdx.z, first = offsets[e];
        T = offsets[e + 1] - first;
        if (t0 >= T) return;
        w += e * matrix_rows * cols;
        x += (int64_t)first * cols;
        y += (int64_t)first * ldy;
    }
    const int ends[kMaxRowGroups] = {end_lo.x, end_lo.y, end_lo.z, end_lo.w, end_hi.x, end_hi.y, end_hi.z, end_hi.w};
    int g = 0;
    if (group_tiles > 0) g = (int)(n0 / 128 / group_tiles);
    else
        while (g < n_groups - 1 && n0 / 128 >= ends[g]) ++g;
    const float* xg = x + (int64_t)g * T * cols;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < cols; k0 += FM_K) {
        for (int i = threadIdx.x; i < FM_TILE * FM_K; i += 256) {
            const int r = i / FM_K, k = i % FM_K;
            ws[k][r] = n0 + r < rows && k0 + k < cols ? w[(n0 + r) * cols + k0 + k] : 0.f;
            xs[k][r] = t0 + r < T && k0 + k < cols ? xg[(int64_t)(t0 + r) * cols + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < FM_K; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[i] = xs[k][ty * 4 + i];
                b[i] = ws[k][tx * 4 + i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + ty * 4 + i;
            const int64_t n = n0 + tx * 4 + j;
            if (t >= T || n >= rows) continue;
            if (to.out == nullptr) {
                const float v = acc[i][j] * scale;
                y[(int64_t)t * ldy + n] = softcap != 0.f ? softcap * tanhf(v / softcap) : v;
                continue;
            }
            const int64_t col = to.column(n);
            if (col >= 0) to.put(to.row(t) + col, to.gate != nullptr ? acc[i][j] * sigmoid_f(to.gate_sum(t, n)) : acc[i][j]);
        }
}

}  // namespace

void launch_row_update(const RowUpdateArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return;
    if (a.n_mix > 0 && (a.x == a.x_out || a.row_index != nullptr)) throw std::runtime_error("launch_row_update: a token shift needs its own output buffer and packed rows");
    if (a.add_bias != nullptr && a.n_add != 1) throw std::runtime_error("launch_row_update: a bias goes with one branch");
    if (a.routed_k > 0 && (a.n_add != 1 || a.add_w[0] == nullptr || a.routed == nullptr)) throw std::runtime_error("launch_row_update: experts' rows go with one normed branch");
    if (a.taps > 0 && (a.x == nullptr || a.x == a.x_out || a.row_index != nullptr || a.n_mix > 0 || a.n_add > 1 || a.add_w[0] != nullptr || a.norm != NormKind::Rms || a.raw.h != nullptr || a.raw.f != nullptr))
        throw std::runtime_error("launch_row_update: a short convolution needs its own output buffer, packed rows, one plain branch and an RMS norm");
    if (a.n_add == 2 && (a.add_w[0] == nullptr || a.add_w[1] == nullptr)) throw std::runtime_error("launch_row_update: two branches are both normed");
    bool vec = a.width % 4 == 0;
    for (int b = 0; b < a.n_add; ++b)
        vec = vec && a.add[b].ld % 4 == 0 && a.add[b].stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a.add[b].p) & 15) == 0;
    if (a.taps > 0) {
        // wide ticks: as many rows per CTA as leave room for two CTAs
        auto fits = [&](int rows) { return (size_t)(rows + a.taps - 1) * a.width * 4 <= (size_t)112 * 1024; };
        if (!vec) launch_conv_rows<1, 1>(a, s);
        else if (a.rows > 512 && fits(8)) launch_conv_rows<4, 8>(a, s);
        else if (a.rows > 256 && fits(4)) launch_conv_rows<4, 4>(a, s);
        else launch_conv_rows<4, 1>(a, s);
        MK_LAUNCH_CHECK();
        return;
    }
    const size_t smem = (size_t)a.width * 4 * (1 + (a.n_mix > 0 ? 1 : 0) + (a.n_add == 2 ? 1 : 0));
    if (smem > (size_t)200 * 1024) throw std::runtime_error("launch_row_update: the model is too wide");
    if (vec) {
        ensure_dynamic_smem(reinterpret_cast<const void*>(&row_update_kernel<4>), smem);
        launch_pdl(row_update_kernel<4>, dim3((unsigned)a.rows), dim3(RU_THREADS), smem, s, a);
    } else {
        ensure_dynamic_smem(reinterpret_cast<const void*>(&row_update_kernel<1>), smem);
        launch_pdl(row_update_kernel<1>, dim3((unsigned)a.rows), dim3(RU_THREADS), smem, s, a);
    }
    MK_LAUNCH_CHECK();
}

void launch_wkv_decay(const Shares& low, int low_col, int rows, int rank, int channels, const float* w2t, const float* w0, float* decay, cudaStream_t s) {
    if (rows <= 0) return;
    if (rows > 256) launch_decay_rows<32>(low, low_col, rows, rank, channels, w2t, w0, decay, s);
    else launch_decay_rows<8>(low, low_col, rows, rank, channels, w2t, w0, decay, s);
}

void launch_channel_gates(const ChannelGatesArgs& a, cudaStream_t s) {
    if (a.lanes.lanes <= 0 || a.longest <= 0) return;
    if (a.dim > CG_COLS) throw std::runtime_error("launch_channel_gates: head dimensions above 256 are not supported");
    if (a.lanes.lanes > 65535 || a.longest > 65535 * 4) throw std::runtime_error("launch_channel_gates: too many lanes or rows");
    if (a.longest > 256) launch_channel_rows<16>(a, s);
    else launch_channel_rows<4>(a, s);
}

void launch_delta_prep(const DeltaPrepArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return;
    if (a.dim > DP_MAX_DIM || a.vdim > DP_MAX_DIM) throw std::runtime_error("launch_delta_prep: head dimensions above 256 are not supported");
    bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.y.ld % 4 == 0 && a.y.stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a.y.p) & 15) == 0;
    for (int c : {a.q_col, a.k_col, a.v_col}) vec = vec && c % 4 == 0;
    const int run = a.rows > 256 ? DP_ROWS : 1;
    const dim3 grid((unsigned)((a.rows + run - 1) / run), (unsigned)((2 * a.kv_heads + a.heads + DP_WARPS - 1) / DP_WARPS));
    if (vec) launch_pdl(delta_prep_kernel<4>, grid, dim3(DP_WARPS * 32), 0, s, a, run);
    else launch_pdl(delta_prep_kernel<1>, grid, dim3(DP_WARPS * 32), 0, s, a, run);
    MK_LAUNCH_CHECK();
}

void launch_head_gate(const float* attn, int rows, int heads, int row_width, int vdim, const Shares& gate, int gate_col, const RowImage& out,
                      cudaStream_t s, const int32_t* row_list, OutputGate kind, float scale) {
    if (rows <= 0) return;
    const int vec_gate = gate_col % 4 == 0 && gate.ld % 4 == 0 && gate.stride % 4 == 0 && (reinterpret_cast<uintptr_t>(gate.p) & 15) == 0 ? 1 : 0;
    launch_pdl(head_gate_kernel, dim3((unsigned)rows), dim3(256), (size_t)heads * 4, s, attn, heads, row_width, vdim, gate, gate_col, out, row_list, kind, vec_gate, scale);
    MK_LAUNCH_CHECK();
}

void launch_side_gate(const Shares& z, int rows, int dim, const uint32_t* ids, const void* table, int table_f32, int64_t table_ld, int slice,
                      const RowImage& out, cudaStream_t s) {
    if (rows <= 0) return;
    launch_pdl(side_gate_kernel, dim3((unsigned)rows), dim3(128), 0, s, z, dim, ids, table, table_f32, table_ld, slice, out);
    MK_LAUNCH_CHECK();
}

void launch_gated_act(const Shares& gu, int rows, int ff, const RowImage& out, cudaStream_t s, const GatedAct& act) {
    if (rows <= 0) return;
    launch_pdl(gated_act_kernel, dim3((unsigned)rows), dim3(256), 0, s, gu, ff, out, act);
    MK_LAUNCH_CHECK();
}

void launch_embed_norm(const EmbedNormArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return;
    const size_t smem = (size_t)a.width * 4;
    if (smem > (size_t)200 * 1024) throw std::runtime_error("launch_embed_norm: the model is too wide");
    ensure_dynamic_smem(reinterpret_cast<const void*>(&embed_norm_kernel), smem);
    launch_pdl(embed_norm_kernel, dim3((unsigned)a.rows), dim3(RU_THREADS), smem, s, a);
    MK_LAUNCH_CHECK();
}

void launch_latent_prep(const LatentPrepArgs& in, cudaStream_t s) {
    LatentPrepArgs a = in;
    if (a.rows <= 0 || (a.q_rank == 0 && a.ff == 0)) return;
    a.lat_vec = a.q_rank % 4 == 0 && a.kv_rank % 4 == 0 && a.q_col % 4 == 0 && a.kv_col % 4 == 0 && a.y.ld % 4 == 0 && a.y.stride % 4 == 0 &&
                (reinterpret_cast<uintptr_t>(a.y.p) & 15) == 0 ? 1 : 0;
    if (a.ff == 0 && a.lat_vec && a.y.n == 1 && a.rows > 256) {
        launch_pdl(latent_rows_kernel, dim3((unsigned)((a.rows + LP_THREADS / 32 - 1) / (LP_THREADS / 32))), dim3(LP_THREADS), 0, s, a);
        MK_LAUNCH_CHECK();
        return;
    }
    const size_t smem = (size_t)std::max(a.ff, a.q_rank + a.kv_rank + a.rot_width) * 4;
    if (smem > (size_t)220 * 1024) throw std::runtime_error("launch_latent_prep: the feed-forward or the latents are too wide");
    const bool vec = a.ff % 4 == 0 && a.ff_col % 4 == 0 && a.y.ld % 4 == 0 && a.y.stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a.y.p) & 15) == 0;
    const dim3 grid((unsigned)a.rows, a.q_rank > 0 && a.ff > 0 ? 2u : 1u);
    auto* kernel = vec ? latent_prep_kernel<4> : latent_prep_kernel<1>;
    ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), smem);
    launch_pdl(kernel, grid, dim3(LP_THREADS), smem, s, a);
    MK_LAUNCH_CHECK();
}

void launch_f32_matmul(const float* w, int64_t rows, int cols, const float* x, int T, float* y, int ldy, int n_groups, const int* group_end,
                       cudaStream_t s, int group_tiles, float scale, const MatmulScatter* to, float softcap) {
    if (T <= 0) return;
    int e[kMaxRowGroups] = {};
    for (int g = 0; g < n_groups && n_groups > 1 && group_tiles == 0; ++g) e[g] = group_end[g];
    const dim3 grid((unsigned)((rows + FM_TILE - 1) / FM_TILE), (unsigned)((T + FM_TILE - 1) / FM_TILE));
    launch_pdl(f32_matmul_kernel, grid, dim3(256), 0, s, w, rows, cols, x, T, y, ldy, scale, softcap, n_groups, group_tiles, make_int4(e[0], e[1], e[2], e[3]),
               make_int4(e[4], e[5], e[6], e[7]), to != nullptr ? *to : MatmulScatter{}, nullptr, (int64_t)0);
    MK_LAUNCH_CHECK();
}

void launch_f32_matmul_experts(const float* w, int experts, const int32_t* offsets, int64_t rows, int64_t matrix_rows, int cols, const float* x, int T, float* y,
                               int ldy, cudaStream_t s) {
    if (T <= 0) return;
    const dim3 grid((unsigned)((rows + FM_TILE - 1) / FM_TILE), (unsigned)((T + FM_TILE - 1) / FM_TILE), (unsigned)experts);
    launch_pdl(f32_matmul_kernel, grid, dim3(256), 0, s, w, rows, cols, x, T, y, ldy, 1.f, 0.f, 1, 0, int4{}, int4{}, MatmulScatter{}, offsets, matrix_rows);
    MK_LAUNCH_CHECK();
}

}  // namespace mk
