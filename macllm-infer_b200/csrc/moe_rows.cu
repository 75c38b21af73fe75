// See moe_rows.h.
//
// A token's choices take their places among their expert's rows by counting up; where those rows begin follows from the counts when
// the rows are gathered.  So two launches route and group a tick of any size.  Places depend on the order in which tokens come to
// count, results do not: a row meets its expert's matrix wherever it lies.
#include "moe_rows.h"
#include "kernels.h"
#include <climits>
#include <type_traits>

namespace mk {

namespace {

constexpr int MR_MAX_EXPERTS = 1024;
constexpr int MR_MAX_TOP = 32;
constexpr int MR_THREADS = 256;

// One token by one warp, PER experts per lane; logit(e) is valid up to `experts` (the shared expert's gate).
template <int PER, typename Logit>
__device__ __forceinline__ void route_token(Logit logit, int t, int experts, int k, const MoeRows& r, int half, int32_t* status, int lane) {
    float v[PER];
    bool bad = false;
#pragma unroll
    for (int c = 0; c < PER; ++c) {
        const int e = lane + 32 * c;
        v[c] = e < experts ? logit(e) : -INFINITY;
        if (e < experts && !isfinite(v[c])) {
            bad = true;
            v[c] = -3.402823466e38f;
        }
    }
    if (lane == 0 && r.shared_gate != nullptr) r.shared_gate[t] = sigmoid_f(logit(experts));
    if (__any_sync(0xffffffffu, bad) && lane == 0) atomicCAS(status, 0, kMoeRouteStatus | (t & 0xFFFF));
    float my_logit = 0.f;
    int mine = 0;        // lane i keeps choice i
    for (int i = 0; i < k; ++i) {
        float bv = -INFINITY;
        int be = INT_MAX;
#pragma unroll
        for (int c = 0; c < PER; ++c)
            if (v[c] > bv) {
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
#pragma unroll
        for (int c = 0; c < PER; ++c)
            if (be == lane + 32 * c) v[c] = -INFINITY;
        if (lane == i) {
            my_logit = bv;
            mine = be;
        }
    }
    if (lane < k) {
        const int64_t p = (int64_t)t * k + lane;
        r.sel[p] = mine;
        r.weight[p] = sigmoid_f(my_logit);
        r.rank[p] = atomicAdd(r.count + half * r.counts + mine, 1);
    }
}

template <int PER>
__global__ void __launch_bounds__(128) moe_route_rows_kernel(Shares logits, int T, int experts, int k, MoeRows r, int half, int32_t* status) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (t >= T) return;
    route_token<PER>([&](int e) { return logits.at(t, e); }, t, experts, k, r, half, status, threadIdx.x & 31);
}

// Eight neighbouring columns.
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        v[2 * i] = __uint_as_float(w[i] << 16);
        v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}

constexpr int MR_ROUTER_THREADS = 512;

// One CTA per token: a warp takes four router rows at once, then the first warp routes.  Shared memory: experts + 4 logits.
template <typename W, int PER>
__global__ void __launch_bounds__(MR_ROUTER_THREADS) moe_router_kernel(RowImage x, const W* __restrict__ w, int experts, int k, MoeRows r, int half,
                                                                       int32_t* status) {
    extern __shared__ float mr_logit[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t t = blockIdx.x;
    const int ld = x.ld, rows = experts + (r.shared_gate != nullptr ? 1 : 0);
    const W* row;
    if constexpr (sizeof(W) == 2) row = x.h + t * ld;
    else row = x.f + t * ld;
    pdl_trigger();
    pdl_wait();
    for (int e = warp * 4; e < rows; e += MR_ROUTER_THREADS / 32 * 4) {
        const W* we[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) we[i] = w + (int64_t)min(e + i, rows - 1) * ld;
        float sum[4] = {};
#pragma unroll 4
        for (int c = lane * 8; c < ld; c += 256) {  // ld is a multiple of 64
            float a[8], b[4][8];
            load8(row + c, a);
#pragma unroll
            for (int i = 0; i < 4; ++i) load8(we[i] + c, b[i]);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 8; ++j) sum[i] = fmaf(a[j], b[i][j], sum[i]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            sum[i] = warp_sum(sum[i]);
            if (lane == 0) mr_logit[e + i] = sum[i];
        }
    }
    __syncthreads();
    if (warp == 0) route_token<PER>([&](int e) { return mr_logit[e]; }, (int)t, experts, k, r, half, status, lane);
}

// One CTA per token.
__global__ void __launch_bounds__(MR_THREADS) moe_gather_kernel(const uint4* x, int experts, int k, int64_t chunks, MoeRows r, int half, uint4* out) {
    __shared__ int at[MR_MAX_TOP];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t t = blockIdx.x;
    pdl_trigger();
    pdl_wait();
    const int32_t* count = r.count + half * r.counts;
    for (int j = warp; j < k; j += MR_THREADS / 32) {
        const int64_t p = t * k + j;
        const int e = r.sel[p];
        int before = 0;
        for (int i = lane; i < e; i += 32) before += count[i];
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
        if (lane == 0) {
            const int pos = before + r.rank[p];
            at[j] = pos;
            r.pos_of_pair[p] = pos;
            r.weight_of_pos[pos] = r.weight[p];
        }
    }
    if (t == 0 && warp == MR_THREADS / 32 - 1) {  // where every expert's rows begin; the other half of the counts for the next call
        int carry = 0;
        for (int base = 0; base < experts; base += 32) {
            const int e = base + lane, c = e < experts ? count[e] : 0;
            int inc = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, inc, o);
                if (lane >= o) inc += v;
            }
            if (e < experts) r.offsets[e] = carry + inc - c;
            carry += __shfl_sync(0xffffffffu, inc, 31);
        }
        if (lane == 0) r.offsets[experts] = carry;
        for (int e = lane; e < r.counts; e += 32) r.count[(half ^ 1) * r.counts + e] = 0;
    }
    __syncthreads();
    for (int64_t c = threadIdx.x; c < chunks; c += MR_THREADS) {
        const uint4 v = x[t * chunks + c];
        for (int j = 0; j < k; ++j) out[at[j] * chunks + c] = v;
    }
}

void check(int experts, int k) {
    if (experts <= 0 || experts > MR_MAX_EXPERTS || k <= 0 || k > MR_MAX_TOP || k > experts) throw std::runtime_error("mixture of experts: at most 1024 experts and 32 choices");
}

// fn(constant): experts per lane of a routing warp.
template <typename Fn>
void per_lane(int experts, Fn fn) {
    if (experts <= 32) fn(std::integral_constant<int, 1>{});
    else if (experts <= 64) fn(std::integral_constant<int, 2>{});
    else if (experts <= 128) fn(std::integral_constant<int, 4>{});
    else if (experts <= 256) fn(std::integral_constant<int, 8>{});
    else fn(std::integral_constant<int, MR_MAX_EXPERTS / 32>{});
}

}  // namespace

void launch_moe_route(const Shares& logits, int T, int experts, int k, const MoeRows& rows, int half, int32_t* status, cudaStream_t s) {
    if (T <= 0) return;
    check(experts, k);
    per_lane(experts, [&](auto per) {
        launch_pdl(moe_route_rows_kernel<per.value>, dim3((unsigned)((T + 3) / 4)), dim3(128), 0, s, logits, T, experts, k, rows, half, status);
    });
    MK_LAUNCH_CHECK();
}

bool moe_router_is_narrow(int T, int experts, int cols) { return T <= 64 && (int64_t)(experts + 1) * cols <= (int64_t)320 * 1024; }

void launch_moe_router(const RowImage& x, const void* w, int T, int experts, int k, const MoeRows& rows, int half, int32_t* status, cudaStream_t s) {
    if (T <= 0) return;
    check(experts, k);
    const size_t smem = (size_t)(experts + 8) * 4;
    const dim3 grid((unsigned)T), block(MR_ROUTER_THREADS);
    per_lane(experts, [&](auto per) {
        if (x.h != nullptr)
            launch_pdl(moe_router_kernel<__nv_bfloat16, per.value>, grid, block, smem, s, x, static_cast<const __nv_bfloat16*>(w), experts, k, rows, half, status);
        else
            launch_pdl(moe_router_kernel<float, per.value>, grid, block, smem, s, x, static_cast<const float*>(w), experts, k, rows, half, status);
    });
    MK_LAUNCH_CHECK();
}

void launch_moe_gather(const void* x, int T, int experts, int k, int64_t bytes, const MoeRows& rows, int half, void* out, cudaStream_t s) {
    if (T <= 0) return;
    if (bytes % 16 != 0) throw std::runtime_error("launch_moe_gather: rows must be multiples of 16 bytes");
    launch_pdl(moe_gather_kernel, dim3((unsigned)T), dim3(MR_THREADS), 0, s, static_cast<const uint4*>(x), experts, k, bytes / 16, rows, half, static_cast<uint4*>(out));
    MK_LAUNCH_CHECK();
}

}  // namespace mk
