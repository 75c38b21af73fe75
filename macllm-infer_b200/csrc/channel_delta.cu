// The delta rule with a decay and a removal rate per key channel (see ChannelDeltaArgs), from the raw projections.  State layout as in
// linear_state.h.
//
// channel_delta_step_kernel: ticks of one-token lanes, a CTA per (head, lane).  The head's state and the low-rank matrix of its decays
// are requested before the predecessor is waited for.  Both sums over the keys run over the old state S,
//   m = k^T S,  o = (r w)^T S - (r . b) m + (r . k) v,  S' = diag(w) S - b m + k v^T   (b: the removal vector),
// folded together over the lanes of a column; the same CTA norms and gates the head.
#include "linear_state.h"
#include "device_util.h"
#include <algorithm>

namespace mk {

namespace {

__device__ __forceinline__ uint32_t cd_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cd_copy16(void* dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(cd_smem(dst)), "l"(src) : "memory"); }
__device__ __forceinline__ float cd_f(float v) { return v; }
__device__ __forceinline__ float cd_f(__nv_bfloat16 v) { return __bfloat162float(v); }

// ------------------------------------------------------------------------------------------------ one-token lanes

constexpr int CS_THREADS = 256;
constexpr int CS_WARPS = CS_THREADS / 32;

template <int KD>
struct DeltaStep {
    static constexpr int LPC = KD / 4;                       // lanes of a column, four keys each
    static constexpr int CPW = 32 / LPC;                     // columns a warp holds side by side
    static constexpr int SLOTS = KD / CS_WARPS / CPW;        // columns of a lane
    static constexpr int PARTS = CS_THREADS / KD;            // threads that share a channel's low-rank sum
    // vectors of the head (r, k, w, b, rw, v, gate, norm, and the two sums per column), the parts, the low-rank input, the decays' matrix
    static size_t bytes(int rank, int esz) { return (size_t)(10 + PARTS) * KD * 4 + (size_t)(rank + 3) / 4 * 16 + (size_t)rank * KD * esz; }
};

template <int KD, typename W2>
__global__ void __launch_bounds__(CS_THREADS, 2) channel_delta_step_kernel(const __grid_constant__ ChannelDeltaArgs a, const W2* w2t, int vec) {
    using P = DeltaStep<KD>;
    constexpr int LPC = P::LPC, CPW = P::CPW, SLOTS = P::SLOTS, PARTS = P::PARTS;
    extern __shared__ __align__(16) float cs_smem[];
    float *s_r = cs_smem, *s_k = s_r + KD, *s_w = s_k + KD, *s_b = s_w + KD, *s_rw = s_b + KD, *s_v = s_rw + KD, *s_g = s_v + KD, *s_nw = s_g + KD, *s_m = s_nw + KD,
          *s_q = s_m + KD, *s_part = s_q + KD, *s_z = s_part + PARTS * KD;
    W2* s_w2 = reinterpret_cast<W2*>(s_z + (a.rank + 3) / 4 * 4);
    __shared__ float red[3][CS_WARPS];
    const LinearStateArgs& c = a.common;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lk = lane & (LPC - 1), lc = lane / LPC;
    const int head = blockIdx.x, dim = c.dim, h0 = head * dim;
    const int64_t channels = (int64_t)c.heads * dim;

    pdl_trigger();
    const StateLane sl = c.lanes.at(blockIdx.y);
    float4 S[SLOTS];
    const float4* src = reinterpret_cast<const float4*>(c.state + ((int64_t)sl.in * c.heads + head) * dim * KD);
#pragma unroll
    for (int s = 0; s < SLOTS; ++s) {
        const int col = (warp * SLOTS + s) * CPW + lc;
        S[s] = sl.in >= 0 && col < dim ? __ldcs(src + (int64_t)col * (KD / 4) + lk) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (vec) {
        constexpr int N = 16 / (int)sizeof(W2);
        const int per = dim / N;
        for (int i = tid; i < a.rank * per; i += CS_THREADS) {
            const int j = i / per, d = (i - j * per) * N;
            cd_copy16(s_w2 + j * KD + d, w2t + j * channels + h0 + d);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    } else {
        for (int i = tid; i < a.rank * dim; i += CS_THREADS) {
            const int j = i / dim, d = i - j * dim;
            s_w2[j * KD + d] = w2t[j * channels + h0 + d];
        }
    }
    float w0 = 0.f, a_bias = 0.f;  // of the thread's channel
    if (tid < dim) {
        w0 = a.w0[h0 + tid];
        a_bias = a.a_bias[h0 + tid];
        s_nw[tid] = c.norm_w[(c.norm_per_head ? h0 : 0) + tid];
    }
    pdl_wait();

    const int64_t row = sl.first;
    // r, k, v, the removal rate and the gate, then the low-rank input
    for (int i = tid; i < 5 * KD; i += CS_THREADS) {
        const int what = i / KD, d = i - what * KD;
        const int col = what == 0 ? a.r_col : (what == 1 ? a.k_col : (what == 2 ? a.v_col : (what == 3 ? a.a_col : c.gate_col)));
        float* dst = what == 0 ? s_r : (what == 1 ? s_k : (what == 2 ? s_v : (what == 3 ? s_b : s_g)));
        dst[d] = d < dim ? a.y.at(row, col + h0 + d) : 0.f;
    }
    for (int j = tid; j < a.rank; j += CS_THREADS) s_z[j] = tanhf(a.y.at(row, a.low_col + j));
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    {
        const int d = tid % KD, part = tid / KD;
        float acc = 0.f;
        if (d < dim)
#pragma unroll 8
            for (int j = part; j < a.rank; j += PARTS) acc = fmaf(s_z[j], cd_f(s_w2[j * KD + d]), acc);
        s_part[part * KD + d] = acc;
    }
    __syncthreads();
    if (tid < KD) {
        float kk = 0.f;
#pragma unroll
        for (int d = lane; d < KD; d += 32) kk = fmaf(s_k[d], s_k[d], kk);
        kk = warp_sum(kk);
        float w = 0.f, b = 0.f;
        const float r = s_r[tid], k = s_k[tid];
        if (tid < dim) {
            float acc = w0;
#pragma unroll
            for (int p = 0; p < PARTS; ++p) acc += s_part[p * KD + tid];
            w = channel_decay_f(acc);
            b = sigmoid_f(s_b[tid] + a_bias) * k / (kk + 1e-6f);
        }
        s_w[tid] = w;
        s_b[tid] = b;
        s_rw[tid] = r * w;
        const float rb = warp_sum(r * b), rk = warp_sum(r * k);
        if (lane == 0) {
            red[0][warp] = rb;
            red[1][warp] = rk;
        }
    }
    __syncthreads();

    const float4 k4 = reinterpret_cast<const float4*>(s_k)[lk], q4 = reinterpret_cast<const float4*>(s_rw)[lk];
    float part[2 * SLOTS];
#pragma unroll
    for (int s = 0; s < SLOTS; ++s) {
        part[s] = fmaf(S[s].x, k4.x, fmaf(S[s].y, k4.y, fmaf(S[s].z, k4.z, S[s].w * k4.w)));
        part[SLOTS + s] = fmaf(S[s].x, q4.x, fmaf(S[s].y, q4.y, fmaf(S[s].z, q4.z, S[s].w * q4.w)));
    }
    int first;
    const int held = fold_lanes<2 * SLOTS, LPC>(part, lane, first);
#pragma unroll
    for (int i = 0; i < 2 * SLOTS; ++i)
        if (i < held) {  // lanes that share a column write the same number
            const int v = first + i;
            (v < SLOTS ? s_m : s_q)[(warp * SLOTS + v % SLOTS) * CPW + lc] = part[i];
        }
    __syncwarp();
    const float4 w4 = reinterpret_cast<const float4*>(s_w)[lk], b4 = reinterpret_cast<const float4*>(s_b)[lk];
    float4* dst = reinterpret_cast<float4*>(c.state + ((int64_t)sl.out * c.heads + head) * dim * KD);
#pragma unroll
    for (int s = 0; s < SLOTS; ++s) {
        const int col = (warp * SLOTS + s) * CPW + lc;
        if (col >= dim) continue;
        const float m = -s_m[col], v = s_v[col];
        __stcs(dst + (int64_t)col * (KD / 4) + lk,
               make_float4(fmaf(b4.x, m, fmaf(w4.x, S[s].x, k4.x * v)), fmaf(b4.y, m, fmaf(w4.y, S[s].y, k4.y * v)), fmaf(b4.z, m, fmaf(w4.z, S[s].z, k4.z * v)),
                           fmaf(b4.w, m, fmaf(w4.w, S[s].w, k4.w * v))));
    }
    __syncthreads();

    float o = 0.f;
    if (tid < KD) {
        float rb = 0.f, rk = 0.f;
#pragma unroll
        for (int w = 0; w < KD / 32; ++w) {
            rb += red[0][w];
            rk += red[1][w];
        }
        if (tid < dim) o = fmaf(-rb, s_m[tid], fmaf(rk, s_v[tid], s_q[tid]));
        const float ss = warp_sum(o * o);
        if (lane == 0) red[2][warp] = ss;
    }
    __syncthreads();
    if (tid < dim) {
        float ss = 0.f;
#pragma unroll
        for (int w = 0; w < KD / 32; ++w) ss += red[2][w];
        const float g = s_g[tid];
        c.image.put(row, h0 + tid, o / sqrtf(ss / (float)dim + c.eps) * s_nw[tid] * (c.gate_sigmoid ? sigmoid_f(g) : silu_f(g)) * c.out_scale);
    }
    if (head == c.heads - 1)
        for (int x = (int)channels + tid; x < c.image.end(); x += CS_THREADS) c.image.put(row, x, 0.f);
}

template <int KD, typename W2>
void launch_step(const ChannelDeltaArgs& a, const W2* w2t, cudaStream_t s) {
    const size_t smem = DeltaStep<KD>::bytes(a.rank, (int)sizeof(W2));
    const int dim = a.common.dim, vec = dim * (int)sizeof(W2) % 16 == 0 ? 1 : 0;
    auto* kernel = channel_delta_step_kernel<KD, W2>;
    ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), smem);
    launch_pdl(kernel, dim3((unsigned)a.common.heads, (unsigned)a.common.lanes.lanes), dim3(CS_THREADS), smem, s, a, w2t, vec);
    MK_LAUNCH_CHECK();
}

template <typename W2>
void launch_step_dim(const ChannelDeltaArgs& a, const W2* w2t, cudaStream_t s) {
    switch (linear_state_key_pad(a.common.dim)) {
        case 32: launch_step<32>(a, w2t, s); break;
        case 64: launch_step<64>(a, w2t, s); break;
        default: launch_step<128>(a, w2t, s); break;
    }
}

}  // namespace

bool channel_delta_can_step(int dim, int rank) { return dim <= 128 && rank <= 256; }

void launch_channel_delta_step(const ChannelDeltaArgs& a, cudaStream_t s) {
    if (a.common.lanes.lanes <= 0) return;
    if (!channel_delta_can_step(a.common.dim, a.rank) || a.common.dim != a.common.vdim || !(a.common.image.h != nullptr || a.common.image.f != nullptr))
        throw std::runtime_error("delta-rule step with channel gates: square heads up to 128, a low rank up to 256, a finished output");
    if (a.common.lanes.lanes > 65535) throw std::runtime_error("delta-rule step with channel gates: at most 65535 lanes");
    if (a.w2h != nullptr) launch_step_dim(a, a.w2h, s);
    else launch_step_dim(a, a.w2t, s);
}

}  // namespace mk
