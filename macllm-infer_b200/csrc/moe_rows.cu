// See moe_rows.h.
//
// Narrow ticks route and group in one CTA: a warp takes a token, the choices stay in shared memory, a counting sort gives every
// pair its row.  Wide ticks route with a warp per token over the whole GPU and group with moe_group_kernel.
#include "moe_rows.h"
#include "kernels.h"
#include <climits>

namespace mk {

namespace {

constexpr int MR_MAX_EXPERTS = 1024;
constexpr int MR_PAIRS = 1024;    // pairs of a tick that one CTA routes and groups
constexpr int MR_MAX_TOP = 32;

// One token by one warp: fn(choice, expert, weight) from lane 0, best first.
template <typename Fn>
__device__ __forceinline__ void route_token(const Shares& logits, int t, int experts, int k, float* shared_gate, int32_t* status, int lane, Fn fn) {
    float v[MR_MAX_EXPERTS / 32];
    int cnt = 0;
    bool bad = false;
    for (int e = lane; e < experts; e += 32) {
        float x = logits.at(t, e);
        if (!isfinite(x)) {
            bad = true;
            x = -3.402823466e38f;
        }
        v[cnt++] = x;
    }
    if (lane == 0 && shared_gate != nullptr) shared_gate[t] = sigmoid_f(logits.at(t, experts));
    if (__any_sync(0xffffffffu, bad) && lane == 0) atomicCAS(status, 0, kMoeRouteStatus | (t & 0xFFFF));
    unsigned taken = 0;  // bit c: this lane's c-th expert was chosen
    for (int i = 0; i < k; ++i) {
        float bv = -INFINITY;
        int be = INT_MAX;
        for (int c = 0; c < cnt; ++c)
            if (!(taken >> c & 1u) && v[c] > bv) {
                bv = v[c];
                be = lane + 32 * c;
            }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oe = __shfl_xor_sync(0xffffffffu, be, o);
            if (ov > bv || (ov == bv && oe < be)) {
                bv = ov;
                be = oe;
            }
        }
        if ((be & 31) == lane) taken |= 1u << (be >> 5);
        if (lane == 0) fn(i, be, sigmoid_f(bv));
    }
}

__global__ void __launch_bounds__(128) moe_route_rows_kernel(Shares logits, int T, int experts, int k, MoeRows r, int32_t* status) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (t >= T) return;
    route_token(logits, t, experts, k, r.shared_gate, status, threadIdx.x & 31, [&](int i, int e, float w) {
        r.sel[(int64_t)t * k + i] = e;
        r.weight[(int64_t)t * k + i] = w;
    });
}

__global__ void __launch_bounds__(1024) moe_route_group_kernel(Shares logits, int T, int experts, int k, MoeRows r, int32_t* status) {
    __shared__ int32_t sel[MR_PAIRS], count[MR_MAX_EXPERTS], start[MR_MAX_EXPERTS + 1];
    __shared__ float weight[MR_PAIRS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pairs = T * k;
    for (int e = threadIdx.x; e < experts; e += 1024) count[e] = 0;
    pdl_trigger();
    pdl_wait();
    __syncthreads();
    for (int t = warp; t < T; t += 32)
        route_token(logits, t, experts, k, r.shared_gate, status, lane, [&](int i, int e, float w) {
            sel[t * k + i] = e;
            weight[t * k + i] = w;
            atomicAdd(&count[e], 1);
        });
    __syncthreads();
    if (warp == 0) {  // exclusive scan, 32 experts at a time
        int carry = 0;
        for (int base = 0; base < experts; base += 32) {
            const int e = base + lane, c = e < experts ? count[e] : 0;
            int inc = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int x = __shfl_up_sync(0xffffffffu, inc, o);
                if (lane >= o) inc += x;
            }
            if (e < experts) start[e] = carry + inc - c;
            carry += __shfl_sync(0xffffffffu, inc, 31);
        }
        if (lane == 0) start[experts] = carry;
    }
    __syncthreads();
    for (int e = threadIdx.x; e <= experts; e += 1024) r.offsets[e] = start[e];
    for (int p = threadIdx.x; p < pairs; p += 1024) {
        r.sel[p] = sel[p];
        r.weight[p] = weight[p];
    }
    // a pair's place among its expert's pairs is the number of earlier ones
    const unsigned below = (1u << lane) - 1u;
    for (int e = warp; e < experts; e += 32) {
        int pos = start[e];
        if (count[e] == 0) continue;
        for (int base = 0; base < pairs; base += 32) {
            const int p = base + lane;
            const bool mine = p < pairs && sel[p] == e;
            const unsigned m = __ballot_sync(0xffffffffu, mine);
            if (mine) {
                const int at = pos + __popc(m & below);
                r.pos_of_pair[p] = at;
                r.token_of_pos[at] = p / k;
            }
            pos += __popc(m);
        }
    }
}

__global__ void __launch_bounds__(128) moe_gather_kernel(const uint4* x, int k, int64_t chunks, MoeRows r, uint4* out) {
    pdl_trigger();
    pdl_wait();
    const int64_t p = blockIdx.x, at = r.pos_of_pair[p], t = p / k;
    for (int64_t c = threadIdx.x; c < chunks; c += 128) out[at * chunks + c] = x[t * chunks + c];
    if (threadIdx.x == 0) r.weight_of_pos[at] = r.weight[p];
}

}  // namespace

int launch_moe_rows(const Shares& logits, int T, int experts, int k, const MoeRows& rows, int32_t* status, cudaStream_t s) {
    if (T <= 0) return 0;
    if (experts > MR_MAX_EXPERTS || k > MR_MAX_TOP || k > experts) throw std::runtime_error("launch_moe_rows: at most 1024 experts and 32 choices");
    if (T * k <= MR_PAIRS) {
        launch_pdl(moe_route_group_kernel, dim3(1), dim3(1024), 0, s, logits, T, experts, k, rows, status);
        MK_LAUNCH_CHECK();
        return 1;
    }
    launch_pdl(moe_route_rows_kernel, dim3((unsigned)((T + 3) / 4)), dim3(128), 0, s, logits, T, experts, k, rows, status);
    MK_LAUNCH_CHECK();
    launch_moe_group(rows.sel, T, k, experts, rows.offsets, rows.pos_of_pair, rows.token_of_pos, s);
    return 2;
}

void launch_moe_gather(const void* x, int T, int k, int64_t bytes, const MoeRows& rows, void* out, cudaStream_t s) {
    if (T <= 0) return;
    if (bytes % 16 != 0) throw std::runtime_error("launch_moe_gather: rows must be multiples of 16 bytes");
    launch_pdl(moe_gather_kernel, dim3((unsigned)(T * k)), dim3(128), 0, s, static_cast<const uint4*>(x), k, bytes / 16, rows, static_cast<uint4*>(out));
    MK_LAUNCH_CHECK();
}

}  // namespace mk
