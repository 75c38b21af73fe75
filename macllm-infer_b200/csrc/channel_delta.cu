// The delta rule with a decay and a removal rate per key channel (see ChannelDeltaArgs), from the raw projections.  State layout as in
// linear_state.h.
//
// channel_delta_step_kernel: ticks of one-token lanes, a CTA per (head, lane).  The head's state and the low-rank matrix of its decays
// are requested before the predecessor is waited for.  Both sums over the keys run over the old state S,
//   m = k^T S,  o = (r w)^T S - (r . b) m + (r . k) v,  S' = diag(w) S - b m + k v^T   (b: the removal vector),
// folded together over the lanes of a column; the same CTA norms and gates the head.
//
// channel_delta_chunk_kernel and channel_delta_states_kernel: prompts, 64 rows at a time, tensor cores.  With L_t the running sum of
// the log decays of a chunk (per channel), u the unit keys, a the removal rates, exponentials per channel,
//   U_t = (u_t e^L_{t-1})^T S_0 + sum_{s<t} (u_t e^{L_{t-1}-L_s} . k_s) v_s - (u_t e^{L_{t-1}-L_s} . a_s u_s) U_s
// are the rows that the removals take off, a triangular system in the chunk's own rows.  Its solution is linear in the state S_0 the
// chunk starts from, and so are the outputs and the state behind the chunk:
//   o = X S_0 + Y,   S = e^L_last S_0 - M S_0 + N.
// X, Y, M and N do not depend on the state: the first kernel makes them for all chunks at once.  The second one walks the chunks of a
// head, 32 value columns per CTA, and has one product per chunk between a state and the next.  The exponents are taken against the
// middle row of the chunk (a decay is at least exp(-exp(-1/2)), so that nothing leaves the range of a float), and every operand that
// is not a bfloat16 number enters as the sum of two (16 bits and more); sums and states are f32.
#include "linear_state.h"
#include "device_util.h"
#include "mma_bf16.cuh"
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
    // r, k, v, the removal rate and the gate, and the low-rank input: all of a thread's numbers share by share, so that their loads overlap
    constexpr int NV = (5 * KD + CS_THREADS - 1) / CS_THREADS;
    {
        const float* y = a.y.p + row * a.y.ld;
        int col[NV + 1];
        float val[NV + 1];
#pragma unroll
        for (int q = 0; q < NV; ++q) {
            const int i = q * CS_THREADS + tid, what = i / KD, d = i - what * KD;
            const int from = what == 0 ? a.r_col : (what == 1 ? a.k_col : (what == 2 ? a.v_col : (what == 3 ? a.a_col : c.gate_col)));
            col[q] = what < 5 && d < dim ? from + h0 + d : -1;
        }
        col[NV] = tid < a.rank ? a.low_col + tid : -1;
#pragma unroll
        for (int q = 0; q <= NV; ++q) val[q] = col[q] >= 0 ? y[col[q]] : 0.f;
#pragma unroll 4
        for (int s = 1; s < a.y.n; ++s)
#pragma unroll
            for (int q = 0; q <= NV; ++q)
                if (col[q] >= 0) val[q] += y[s * a.y.stride + col[q]];
#pragma unroll
        for (int q = 0; q < NV; ++q) {
            const int i = q * CS_THREADS + tid, what = i / KD, d = i - what * KD;
            if (what < 5) (what == 0 ? s_r : (what == 1 ? s_k : (what == 2 ? s_v : (what == 3 ? s_b : s_g))))[d] = val[q];
        }
        if (tid < a.rank) s_z[tid] = tanhf(val[NV]);
    }
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

// ------------------------------------------------------------------------------------------------ prompts

constexpr int CC_ROWS = 64;        // rows of a chunk
constexpr int CC_WARPS = 16;
constexpr int CC_THREADS = CC_WARPS * 32;
constexpr int CC_SLICE = 32;       // value columns of a CTA of the second kernel
constexpr int CC_AP = CC_ROWS + 8; // padded row of a [row][row] matrix

// What the first kernel leaves for the second, per chunk and head.  M and X are B operands of an m16n8k16 product in the order of its
// fragments: [16 columns][16 inner][part][lane] of 16 bytes; N and Y are accumulator tiles, [16 values][8 columns][lane] of 16 bytes.
template <int KD>
struct ChunkResult {
    static constexpr int M = 0, X = M + KD * KD * 4, N = X + CC_ROWS * KD * 4, Y = N + KD * KD * 4, DECAY = Y + KD * CC_ROWS * 4, BYTES = DECAY + KD * 4;
    static constexpr int TILE = KD / 16 * 2 * 512;   // bytes of 16 columns of M or X
};

template <int KD>
struct ChunkSmem {
    static constexpr int KP = KD + 8;
    static constexpr int OPERAND = CC_ROWS * KP;       // bfloat16 numbers of one part
    static constexpr int TRI = CC_ROWS * CC_AP;
    static constexpr size_t HALVES = (size_t)5 * 2 * OPERAND + 2 * 2 * TRI + 2 * 4 * 16 * 24;
    static constexpr size_t FLOATS = 4 * 16 * 20 + 3 * KD + CC_THREADS;
    static constexpr size_t BYTES = HALVES * 2 + FLOATS * 4;
    static_assert(BYTES <= 227 * 1024, "shared memory");
    static_assert((size_t)CC_ROWS * (KD + 4) * 4 <= (size_t)2 * OPERAND * 2, "the log decays fit in an operand's place");
    static_assert((size_t)3 * TRI + CC_ROWS * KP <= (size_t)4 * OPERAND, "the low-rank operands fit in two operands' places");
};

__device__ __forceinline__ int chunk_slot(const StateLane& sl, int lane, int chunk) { return sl.first / CC_ROWS + lane + chunk; }  // lanes in packed order do not overlap

template <int KD>
__global__ void __launch_bounds__(CC_THREADS, 1) channel_delta_chunk_kernel(const __grid_constant__ ChannelDeltaArgs a, uint8_t* results, int vec) {
    using P = ChunkSmem<KD>;
    using R = ChunkResult<KD>;
    constexpr int KP = P::KP, C = CC_ROWS, AP = CC_AP;
    constexpr int VT = KD / 16, CG = CC_WARPS / VT, NT = KD / 8 / CG, YT = C / 8 / CG, XT = KD / 32;
    extern __shared__ __align__(16) unsigned char cc_raw[];
    __nv_bfloat16* base = reinterpret_cast<__nv_bfloat16*>(cc_raw);
    auto operand = [&](int i) { return Split{base + i * 2 * P::OPERAND, KP, P::OPERAND}; };
    const Split Kq = operand(0), Br = operand(1), Kw = operand(2), Rq = operand(3), V = operand(4);   // Kq becomes W, Kw becomes G
    __nv_bfloat16* tri = base + 10 * P::OPERAND;
    const Split A1{tri, AP, P::TRI}, A2{tri + 2 * P::TRI, AP, P::TRI};
    const Split Ti{tri + 4 * P::TRI, 24, 4 * 16 * 24};
    float* s_diag = reinterpret_cast<float*>(tri + 4 * P::TRI + 2 * 4 * 16 * 24);   // [4][16][20]
    float *s_start = s_diag + 4 * 16 * 20, *s_em = s_start + KD, *s_elm = s_em + KD, *s_sum = s_elm + KD;   // s_sum: [CC_THREADS]
    float* s_l = reinterpret_cast<float*>(V.p);                                     // [C][KD + 4]
    constexpr int LP = KD + 4;

    const LinearStateArgs& cm = a.common;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tq = lane & 3;
    const int head = blockIdx.x, dim = cm.dim, h0 = head * dim;
    pdl_trigger();
    const StateLane sl = cm.lanes.at(blockIdx.z);
    const int chunk = blockIdx.y;
    if (chunk * C >= sl.n) return;
    const int m = min(C, sl.n - chunk * C);
    const int64_t row0 = (int64_t)sl.first + (int64_t)chunk * C, channels = (int64_t)cm.heads * dim;
    uint8_t* out = results + ((int64_t)chunk_slot(sl, blockIdx.z, chunk) * cm.heads + head) * R::BYTES;
    __nv_bfloat16* zs = base;                 // [3][C][AP]
    __nv_bfloat16* w2 = zs + 3 * P::TRI;      // [C][KP]
    // 64 rows of the low-rank matrix; columns past the head and rows past the rank are zeros
    auto request_w2 = [&](int j0) {
        const int nj = min(C, a.rank - j0);
        if (vec && dim % 8 == 0) {
            for (int i = tid; i < C * (KD / 8); i += CC_THREADS) {
                const int j = i / (KD / 8), c = i % (KD / 8) * 8;
                const bool live = j < nj && c < dim;
                mc_cp_async16(w2 + j * KP + c, a.w2h + (live ? (int64_t)(j0 + j) * channels + h0 + c : 0), live);
            }
        } else {
            for (int i = tid; i < C * KD; i += CC_THREADS) {
                const int j = i / KD, c = i % KD;
                w2[j * KP + c] = j < nj && c < dim ? a.w2h[(int64_t)(j0 + j) * channels + h0 + c] : __float2bfloat16_rn(0.f);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    request_w2(0);
    const int quarter = warp >> 2, z16 = (warp & 3) * 16;
    constexpr int ROWS = C / CC_WARPS, EL = KD / 32;   // rows of a warp, channels of a lane
    float w0[XT][2], bias[EL];
#pragma unroll
    for (int j = 0; j < XT; ++j)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int c = quarter * (KD / 4) + j * 8 + 2 * tq + x;
            w0[j][x] = c < dim ? a.w0[h0 + c] : 0.f;
        }
#pragma unroll
    for (int e = 0; e < EL; ++e) bias[e] = lane * EL + e < dim ? a.a_bias[h0 + lane * EL + e] : 0.f;
    pdl_wait();

    // raw projections on their way while the decays are made: keys and queries in the places of operands, rates in the triangles'
    const bool plain = vec && a.y.n == 1;
    float *raw_k = reinterpret_cast<float*>(Kw.p), *raw_r = reinterpret_cast<float*>(Rq.p), *raw_g = reinterpret_cast<float*>(tri);   // [C][KD]
    auto request_raw = [&](float* dst, int col) {
        for (int i = tid; i < C * (KD / 4); i += CC_THREADS) {
            const int t = i / (KD / 4), c = i % (KD / 4) * 4;
            if (plain) {
                const bool live = t < m && c < dim;
                mc_cp_async16(dst + t * KD + c, a.y.p + (live ? (row0 + t) * a.y.ld + col + h0 + c : 0), live);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) dst[t * KD + c + e] = t < m && c + e < dim ? a.y.at(row0 + t, col + h0 + c + e) : 0.f;
            }
        }
    };
    request_raw(raw_k, a.k_col);
    request_raw(raw_r, a.r_col);
    request_raw(raw_g, a.a_col);
    asm volatile("cp.async.commit_group;" ::: "memory");
    // ---- log decays: tanh of the low-rank input (three parts: f32) times w2
    {
        float acc[XT][4] = {};
        const int c0 = quarter * (KD / 4);
        for (int j0 = 0; j0 < a.rank; j0 += C) {
            const int nj = min(C, a.rank - j0);
            if (j0 > 0) {
                __syncthreads();
                request_w2(j0);
            }
            float z[C * C / CC_THREADS];
#pragma unroll
            for (int q = 0; q < C * C / CC_THREADS; ++q) {
                const int i = q * CC_THREADS + tid, t = i / C, j = i % C;
                const int64_t at = (row0 + t) * a.y.ld + a.low_col + j0 + j;
                z[q] = t < m && j < nj ? a.y.p[at] : 0.f;
            }
            for (int p = 1; p < a.y.n; ++p)
#pragma unroll
                for (int q = 0; q < C * C / CC_THREADS; ++q) {
                    const int i = q * CC_THREADS + tid, t = i / C, j = i % C;
                    if (t < m && j < nj) z[q] += a.y.p[p * a.y.stride + (row0 + t) * a.y.ld + a.low_col + j0 + j];
                }
#pragma unroll
            for (int q = 0; q < C * C / CC_THREADS; ++q) {
                const int i = q * CC_THREADS + tid;
                float x = 1.0f - __fdividef(2.0f, 1.0f + __expf(2.0f * z[q]));  // tanh, to a few 1e-7 of 1
#pragma unroll
                for (int p = 0; p < 3; ++p) {
                    const __nv_bfloat16 h = __float2bfloat16_rn(x);
                    zs[p * P::TRI + i / C * AP + i % C] = h;
                    x -= __bfloat162float(h);
                }
            }
            if (j0 == 0) asm volatile("cp.async.wait_group 1;" ::: "memory");
            else asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();
            for (int k = 0; k < (nj + 15) / 16; ++k) {
                uint32_t af[3][4], bf[4];
#pragma unroll
                for (int p = 0; p < 3; ++p) mma_a(af[p], zs + p * P::TRI + z16 * AP + k * 16, AP, lane);
#pragma unroll
                for (int j = 0; j < XT; j += 2) {
                    mma_b_t(bf, w2 + k * 16 * KP + c0 + j * 8, KP, lane);
#pragma unroll
                    for (int p = 0; p < 3; ++p) {
                        mc_mma(acc[j], af[p], bf[0], bf[1]);
                        mc_mma(acc[j + 1], af[p], bf[2], bf[3]);
                    }
                }
            }
        }
#pragma unroll
        for (int j = 0; j < XT; ++j)
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int t = z16 + gid + (x >> 1) * 8, c = c0 + j * 8 + 2 * tq + (x & 1);
                s_l[t * LP + c] = t < m && c < dim ? -0.60653066f * __fdividef(1.0f, 1.0f + __expf(-acc[j][x] - w0[j][x & 1])) : 0.f;
            }
    }
    __syncthreads();
    // ---- running sums over the rows, a part of them per thread, against the middle row; then their exponentials
    constexpr int PARTS = CC_THREADS / KD, PART = C / PARTS;
    {
        const int c = tid % KD, part = tid / KD;
        float l[PART], sum = 0.f;
#pragma unroll
        for (int t = 0; t < PART; ++t) l[t] = sum += s_l[(part * PART + t) * LP + c];
        s_sum[part * KD + c] = sum;
        __syncthreads();
        float before = 0.f, mid = 0.f, all = 0.f;
#pragma unroll
        for (int p = 0; p < PARTS; ++p) {
            const float x = s_sum[p * KD + c];
            if (p < part) before += x;
            if (p < PARTS / 2) mid += x;
            all += x;
        }
#pragma unroll
        for (int t = 0; t < PART; ++t) s_l[(part * PART + t) * LP + c] = expf(l[t] + (before - mid));
        if (part == 0) {
            s_em[c] = expf(mid);
            s_start[c] = expf(-mid);
            s_elm[c] = expf(all - mid);
            reinterpret_cast<float*>(out + R::DECAY)[c] = expf(all);
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // ---- operands: a warp per row; the values on their way meanwhile
    float kr[ROWS][EL], rr[ROWS][EL], gr[ROWS][EL], vr[ROWS][EL];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int t = i * CC_WARPS + warp, c = lane * EL;
        if (plain) {
            const float* src = a.y.p + (t < m && c < dim ? (row0 + t) * a.y.ld + a.v_col + h0 + c : 0);
#pragma unroll
            for (int e = 0; e < EL; e += 2) {
                const float2 v = *reinterpret_cast<const float2*>(src + e);
                vr[i][e] = v.x;
                vr[i][e + 1] = v.y;
            }
        } else {
#pragma unroll
            for (int e = 0; e < EL; ++e) vr[i][e] = t < m && c + e < dim ? a.y.at(row0 + t, a.v_col + h0 + c + e) : 0.f;
        }
#pragma unroll
        for (int e = 0; e < EL; ++e) {
            kr[i][e] = raw_k[t * KD + c + e];
            rr[i][e] = raw_r[t * KD + c + e];
            gr[i][e] = raw_g[t * KD + c + e];
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int t = i * CC_WARPS + warp, c = lane * EL;
        float kk = 0.f;
#pragma unroll
        for (int e = 0; e < EL; ++e) kk = fmaf(kr[i][e], kr[i][e], kk);
        kk = warp_sum(kk);
        const float unit = 1.0f / sqrtf(kk + 1e-6f);
        const float* now = s_l + t * LP + c;
        const float* prev = t == 0 ? s_start + c : now - LP;
        float q[EL], b[EL], w[EL], o[EL];
#pragma unroll
        for (int e = 0; e < EL; ++e) {
            const float l = now[e], later = __fdividef(1.0f, l), u = kr[i][e] * unit;
            q[e] = u * prev[e];
            b[e] = __fdividef(u * later, 1.0f + __expf(-(gr[i][e] + bias[e])));
            w[e] = kr[i][e] * later;
            o[e] = rr[i][e] * l;
        }
#pragma unroll
        for (int e = 0; e < EL; e += 2) {
            Kq.put2(t, c + e, q[e], q[e + 1]);
            Br.put2(t, c + e, b[e], b[e + 1]);
            Kw.put2(t, c + e, w[e], w[e + 1]);
            Rq.put2(t, c + e, o[e], o[e + 1]);
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
#pragma unroll
        for (int e = 0; e < EL; e += 2) {
            const bool live = i * CC_WARPS + warp < m && lane * EL < dim;  // a pack that was not there was read from elsewhere
            V.put2(i * CC_WARPS + warp, lane * EL + e, live ? vr[i][e] : 0.f, live ? vr[i][e + 1] : 0.f);
        }
    // ---- products of the chunk's rows among themselves, 16 x 16 per warp; what lies behind a row is zero
    const int s16 = quarter * 16, r16 = ((warp + (quarter < 2 ? 0 : quarter)) & 3) * 16;  // the tiles that count: two or three per scheduler
    float a_kb[2][4] = {}, a_kk[2][4] = {}, a_rk[2][4] = {}, a_rb[2][4] = {};
    if (s16 <= r16) {
#pragma unroll 2
        for (int k = 0; k < KD / 16; ++k) {
            uint32_t qh[4], ql[4], rh[4], rl[4], bh[4], bl[4], wh[4], wl[4];
            mma_a(qh, Kq.at(r16, k * 16), KP, lane);
            mma_a(ql, Kq.at(r16, k * 16) + Kq.rest, KP, lane);
            mma_a(rh, Rq.at(r16, k * 16), KP, lane);
            mma_a(rl, Rq.at(r16, k * 16) + Rq.rest, KP, lane);
            mma_b(bh, Br.at(s16, k * 16), KP, lane);
            mma_b(bl, Br.at(s16, k * 16) + Br.rest, KP, lane);
            mma_b(wh, Kw.at(s16, k * 16), KP, lane);
            mma_b(wl, Kw.at(s16, k * 16) + Kw.rest, KP, lane);
            mma_split(a_kb[0], a_kb[1], qh, ql, bh, bl);
            mma_split(a_kk[0], a_kk[1], qh, ql, wh, wl);
            mma_split(a_rb[0], a_rb[1], rh, rl, bh, bl);
            mma_split(a_rk[0], a_rk[1], rh, rl, wh, wl);
        }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int t = r16 + gid + (x >> 1) * 8, s = s16 + j * 8 + 2 * tq + (x & 1);
            if (s >= t) a_kb[j][x] = a_kk[j][x] = 0.f;
            if (s > t) a_rk[j][x] = a_rb[j][x] = 0.f;
            if (s16 == r16) s_diag[t * 20 + s - s16] = a_kb[j][x];
        }
    auto put_tile = [&](const Split& to, const float (&v)[2][4]) {
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int h = 0; h < 2; ++h) to.put2(r16 + gid + 8 * h, s16 + j * 8 + 2 * tq, v[j][2 * h], v[j][2 * h + 1]);
    };
    put_tile(A1, a_kb);
    put_tile(A2, a_rk);
    __syncthreads();
    // ---- inverses of the diagonal blocks, a column per lane; meanwhile what the writes alone give
    if (warp < 4 && lane < 16) {
        const float4* d = reinterpret_cast<const float4*>(s_diag + warp * 16 * 20);
        float x[16];
        float4 next[4] = {};
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            const float row[16] = {next[0].x, next[0].y, next[0].z, next[0].w, next[1].x, next[1].y, next[1].z, next[1].w,
                                   next[2].x, next[2].y, next[2].z, next[2].w, next[3].x, next[3].y, next[3].z, next[3].w};
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (i + 1 < 16 && 4 * k < i + 1) next[k] = d[(i + 1) * 5 + k];
            float v[4] = {i == lane ? 1.f : 0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int k = 0; k < i; ++k) v[k & 3] = fmaf(-row[k], x[k], v[k & 3]);
            x[i] = (v[0] + v[1]) + (v[2] + v[3]);
            const __nv_bfloat16 h = __float2bfloat16_rn(x[i]);
            *Ti.at(warp * 16 + i, lane) = h;
            *(Ti.at(warp * 16 + i, lane) + Ti.rest) = __float2bfloat16_rn(x[i] - __bfloat162float(h));
        }
    }
    const int vt = warp % VT * 16, cg = warp / VT;   // 16 values (or keys), a group of columns
    const int t0 = cg * YT * 8, n0 = cg * NT * 8;
    // [16 values from vt on][columns] += (rows' values)^T B over the rows [0, steps * 16)
    auto values_times = [&](const Split& A, int k, uint32_t (&h)[4], uint32_t (&l)[4]) {
        mma_a_t(h, A.at(k * 16, vt), KP, lane);
        mma_a_t(l, A.at(k * 16, vt) + A.rest, KP, lane);
    };
    float y[YT][4] = {}, n[NT][4] = {};
#pragma unroll 1
    for (int k = 0; k < C / 16; ++k) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        values_times(V, k, ah, al);
#pragma unroll
        for (int j = 0; j < YT; j += 2) {
            if (k * 16 > t0 + j * 8) continue;  // these rows come before
            mma_b(bh, A2.at(t0 + j * 8, k * 16), AP, lane);
            mma_b(bl, A2.at(t0 + j * 8, k * 16) + A2.rest, AP, lane);
            mma_split(y[j], y[j + 1], ah, al, bh, bl);
        }
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
            mma_b_t(bh, Kw.at(k * 16, n0 + j * 8), KP, lane);
            mma_b_t(bl, Kw.at(k * 16, n0 + j * 8) + Kw.rest, KP, lane);
            mma_split(n[j], n[j + 1], ah, al, bh, bl);
        }
    }
    __syncthreads();
    put_tile(A2, a_kk);
    __syncthreads();
    // ---- the triangular system, 16 columns of the state's part (W) or of the values' part (G) per warp
    if (warp < 2 * VT) {
        const bool values = warp >= VT;
        const Split to = values ? Kw : Kq;
        const int c16 = (values ? warp - VT : warp) * 16;
#pragma unroll 1
        for (int i = 0; i < C / 16; ++i) {
            float rhs[2][4] = {}, taken[2][4] = {}, x[2][4] = {};
            uint32_t ah[4], al[4], bh[4], bl[4];
            if (values) {
#pragma unroll 1
                for (int k = 0; k <= i; ++k) {
                    mma_a(ah, A2.at(i * 16, k * 16), AP, lane);
                    mma_a(al, A2.at(i * 16, k * 16) + A2.rest, AP, lane);
                    mma_b_t(bh, V.at(k * 16, c16), KP, lane);
                    mma_b_t(bl, V.at(k * 16, c16) + V.rest, KP, lane);
                    mma_split(rhs[0], rhs[1], ah, al, bh, bl);
                }
            } else {
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
                        const float2 v = to.get2(i * 16 + gid + 8 * h, c16 + j * 8 + 2 * tq);
                        rhs[j][2 * h] = v.x;
                        rhs[j][2 * h + 1] = v.y;
                    }
            }
#pragma unroll 1
            for (int k = 0; k < i; ++k) {
                mma_a(ah, A1.at(i * 16, k * 16), AP, lane);
                mma_a(al, A1.at(i * 16, k * 16) + A1.rest, AP, lane);
                mma_b_t(bh, to.at(k * 16, c16), KP, lane);
                mma_b_t(bl, to.at(k * 16, c16) + to.rest, KP, lane);
                mma_split(taken[0], taken[1], ah, al, bh, bl);
            }
            __syncwarp();
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h)
                    to.put2(i * 16 + gid + 8 * h, c16 + j * 8 + 2 * tq, rhs[j][2 * h] - taken[j][2 * h], rhs[j][2 * h + 1] - taken[j][2 * h + 1]);
            __syncwarp();
            mma_a(ah, Ti.at(i * 16, 0), 24, lane);
            mma_a(al, Ti.at(i * 16, 0) + Ti.rest, 24, lane);
            mma_b_t(bh, to.at(i * 16, c16), KP, lane);
            mma_b_t(bl, to.at(i * 16, c16) + to.rest, KP, lane);
            mma_split(x[0], x[1], ah, al, bh, bl);
            __syncwarp();
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h) to.put2(i * 16 + gid + 8 * h, c16 + j * 8 + 2 * tq, x[j][2 * h], x[j][2 * h + 1]);
            __syncwarp();
        }
    }
    __syncthreads();
    put_tile(A2, a_rb);
    __syncthreads();
    const Split W = Kq, G = Kw;
    // two accumulator tiles side by side as one fragment of a B operand
    auto store_pair = [&](int at, const float (&lo_cols)[4], const float (&hi_cols)[4]) {
        uint4 hi, lo;
        mc_split(lo_cols[0], lo_cols[1], hi.x, lo.x);
        mc_split(hi_cols[0], hi_cols[1], hi.y, lo.y);
        mc_split(lo_cols[2], lo_cols[3], hi.z, lo.z);
        mc_split(hi_cols[2], hi_cols[3], hi.w, lo.w);
        *reinterpret_cast<uint4*>(out + at + lane * 16) = hi;
        *reinterpret_cast<uint4*>(out + at + 512 + lane * 16) = lo;
    };
    // ---- values' side: Y and N
#pragma unroll 1
    for (int k = 0; k < C / 16; ++k) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        values_times(G, k, ah, al);
#pragma unroll
        for (int i = 0; i < 4; ++i) {  // taken off
            ah[i] ^= 0x80008000u;
            al[i] ^= 0x80008000u;
        }
#pragma unroll
        for (int j = 0; j < YT; j += 2) {
            if (k * 16 > t0 + j * 8) continue;
            mma_b(bh, A2.at(t0 + j * 8, k * 16), AP, lane);
            mma_b(bl, A2.at(t0 + j * 8, k * 16) + A2.rest, AP, lane);
            mma_split(y[j], y[j + 1], ah, al, bh, bl);
        }
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
            mma_b_t(bh, Br.at(k * 16, n0 + j * 8), KP, lane);
            mma_b_t(bl, Br.at(k * 16, n0 + j * 8) + Br.rest, KP, lane);
            mma_split(n[j], n[j + 1], ah, al, bh, bl);
        }
    }
#pragma unroll
    for (int j = 0; j < YT; ++j)
        *reinterpret_cast<float4*>(out + R::Y + ((vt / 16) * (C / 8) + t0 / 8 + j) * 512 + lane * 16) = make_float4(y[j][0], y[j][1], y[j][2], y[j][3]);
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        const float2 f = *reinterpret_cast<const float2*>(s_elm + n0 + j * 8 + 2 * tq);
        *reinterpret_cast<float4*>(out + R::N + ((vt / 16) * (KD / 8) + n0 / 8 + j) * 512 + lane * 16) =
            make_float4(n[j][0] * f.x, n[j][1] * f.y, n[j][2] * f.x, n[j][3] * f.y);
    }
    // ---- state's side: M, 16 keys x NT tiles per warp, and X, 16 rows x XT tiles
    {
        float mm[NT][4] = {};
#pragma unroll 1
        for (int k = 0; k < C / 16; ++k) {
            uint32_t ah[4], al[4], bh[4], bl[4];
            values_times(Br, k, ah, al);
#pragma unroll
            for (int j = 0; j < NT; j += 2) {
                mma_b_t(bh, W.at(k * 16, n0 + j * 8), KP, lane);
                mma_b_t(bl, W.at(k * 16, n0 + j * 8) + W.rest, KP, lane);
                mma_split(mm[j], mm[j + 1], ah, al, bh, bl);
            }
        }
        const float f0 = s_elm[vt + gid], f1 = s_elm[vt + gid + 8];
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const float2 e = *reinterpret_cast<const float2*>(s_em + n0 + j * 8 + 2 * tq);
            mm[j][0] *= f0 * e.x;
            mm[j][1] *= f0 * e.y;
            mm[j][2] *= f1 * e.x;
            mm[j][3] *= f1 * e.y;
        }
#pragma unroll
        for (int j = 0; j < NT; j += 2) store_pair(R::M + (vt / 16) * R::TILE + (n0 / 8 + j) / 2 * 1024, mm[j], mm[j + 1]);
    }
    {
        float xx[XT][4] = {};
        const int c0 = quarter * (KD / 4), t16 = ((warp + quarter) & 3) * 16;  // as many rows before them for every scheduler
#pragma unroll 1
        for (int k = 0; k < C / 16; ++k) {
            if (k * 16 > t16) continue;
            uint32_t ah[4], al[4], bh[4], bl[4];
            mma_a(ah, A2.at(t16, k * 16), AP, lane);
            mma_a(al, A2.at(t16, k * 16) + A2.rest, AP, lane);
#pragma unroll
            for (int j = 0; j < XT; j += 2) {
                mma_b_t(bh, W.at(k * 16, c0 + j * 8), KP, lane);
                mma_b_t(bl, W.at(k * 16, c0 + j * 8) + W.rest, KP, lane);
                mma_split(xx[j], xx[j + 1], ah, al, bh, bl);
            }
        }
#pragma unroll
        for (int j = 0; j < XT; ++j) {
            const float2 e = *reinterpret_cast<const float2*>(s_em + c0 + j * 8 + 2 * tq);
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const float2 r = Rq.get2(t16 + gid + 8 * h, c0 + j * 8 + 2 * tq);
                xx[j][2 * h] = (r.x - xx[j][2 * h]) * e.x;
                xx[j][2 * h + 1] = (r.y - xx[j][2 * h + 1]) * e.y;
            }
        }
#pragma unroll
        for (int j = 0; j < XT; j += 2) store_pair(R::X + (t16 / 16) * R::TILE + (c0 / 8 + j) / 2 * 1024, xx[j], xx[j + 1]);
    }
}

// Grid (slices of 32 values, heads, lanes); KD / 16 warps carry the state, 16 keys each, four more make the outputs, 16 rows each.
template <int KD>
struct StatesSmem {
    static constexpr int WARPS = KD / 16 + 4, KP = KD + 8;
    static constexpr int STATE = CC_SLICE * KP;   // bfloat16 numbers of one part
    static constexpr size_t BYTES = (size_t)2 * WARPS * ChunkResult<KD>::TILE + (size_t)2 * 2 * STATE * 2;
    static_assert(BYTES <= 227 * 1024, "shared memory");
};

template <int KD>
__global__ void __launch_bounds__(StatesSmem<KD>::WARPS * 32, 1) channel_delta_states_kernel(const __grid_constant__ ChannelDeltaArgs a, const uint8_t* results) {
    using P = StatesSmem<KD>;
    using R = ChunkResult<KD>;
    constexpr int KP = P::KP, STEPS = KD / 16;
    extern __shared__ __align__(16) unsigned char st_raw[];
    const LinearStateArgs& cm = a.common;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tq = lane & 3;
    const int head = blockIdx.y, v0 = blockIdx.x * CC_SLICE, dim = cm.dim;
    const bool carries = warp < STEPS;
    const int tile = carries ? warp : warp - STEPS;    // of M's columns or of X's
    unsigned char* ring = st_raw + (size_t)warp * 2 * R::TILE;
    __nv_bfloat16* states = reinterpret_cast<__nv_bfloat16*>(st_raw + (size_t)P::WARPS * 2 * R::TILE);
    auto state = [&](int i) { return Split{states + (i & 1) * 2 * P::STATE, KP, P::STATE}; };

    pdl_trigger();
    const StateLane sl = cm.lanes.at(blockIdx.z);
    const int chunks = (sl.n + CC_ROWS - 1) / CC_ROWS;
    float S[2][2][4];   // [16 values][8 keys]
    if (carries) {
        const float* src = cm.state + ((int64_t)sl.in * cm.heads + head) * dim * KD;
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int v = v0 + i * 16 + gid + 8 * h;
                    float2 x = make_float2(0.f, 0.f);
                    if (sl.in >= 0 && v < dim) x = *reinterpret_cast<const float2*>(src + (int64_t)v * KD + tile * 16 + j * 8 + 2 * tq);
                    S[i][j][2 * h] = x.x;
                    S[i][j][2 * h + 1] = x.y;
                }
    }
    auto publish = [&](const Split& to) {
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h) to.put2(i * 16 + gid + 8 * h, tile * 16 + j * 8 + 2 * tq, S[i][j][2 * h], S[i][j][2 * h + 1]);
    };
    if (carries) publish(state(0));
    pdl_wait();
    const uint8_t* first = results + ((int64_t)chunk_slot(sl, blockIdx.z, 0) * cm.heads + head) * R::BYTES;
    const int64_t step = (int64_t)cm.heads * R::BYTES;
    auto request = [&](int ch) {
        if (ch < chunks) {
            const uint8_t* src = first + ch * step + (carries ? R::M : R::X) + tile * R::TILE + lane * 16;
            unsigned char* dst = ring + (ch & 1) * R::TILE + lane * 16;
#pragma unroll
            for (int i = 0; i < R::TILE / 512; ++i) cd_copy16(dst + i * 512, src + i * 512);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    request(0);
    for (int ch = 0; ch < chunks; ++ch) {
        __syncwarp();  // the stage that is asked for next was read by the whole warp
        request(ch + 1);
        const uint8_t* res = first + ch * step;
        float4 add[2][2];
        float2 keep[2];
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int vt = v0 / 16 + i;
                add[i][j] = vt >= STEPS ? make_float4(0.f, 0.f, 0.f, 0.f)
                                        : *reinterpret_cast<const float4*>(res + (carries ? R::N + (vt * (KD / 8) + tile * 2 + j) * 512 : R::Y + (vt * (CC_ROWS / 8) + tile * 2 + j) * 512) + lane * 16);
            }
        if (carries)
#pragma unroll
            for (int j = 0; j < 2; ++j) keep[j] = *reinterpret_cast<const float2*>(res + R::DECAY + (tile * 16 + j * 8 + 2 * tq) * 4);
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();  // the state the chunk starts from is there, and the one before it was read
        const Split from = state(ch);
        const uint4* b = reinterpret_cast<const uint4*>(ring + (ch & 1) * R::TILE) + lane;
        float acc[2][2][4] = {};
#pragma unroll
        for (int k = 0; k < STEPS; ++k) {
            const uint4 h4 = b[k * 64], l4 = b[k * 64 + 32];
            const uint32_t bh[4] = {h4.x, h4.y, h4.z, h4.w}, bl[4] = {l4.x, l4.y, l4.z, l4.w};
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                uint32_t ah[4], al[4];
                mma_a(ah, from.at(i * 16, k * 16), KP, lane);
                mma_a(al, from.at(i * 16, k * 16) + from.rest, KP, lane);
                mma_split(acc[i][0], acc[i][1], ah, al, bh, bl);
            }
        }
        if (carries) {
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const float n[4] = {add[i][j].x, add[i][j].y, add[i][j].z, add[i][j].w};
#pragma unroll
                    for (int x = 0; x < 4; ++x) S[i][j][x] = fmaf((x & 1) ? keep[j].y : keep[j].x, S[i][j][x], n[x] - acc[i][j][x]);
                }
            publish(state(ch + 1));
        } else {
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const int t = ch * CC_ROWS + tile * 16 + j * 8 + 2 * tq + x;
                    if (t >= sl.n) continue;
                    float* o = cm.out + ((int64_t)(sl.first + t) * cm.heads + head) * dim;
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        const float y[4] = {add[i][j].x, add[i][j].y, add[i][j].z, add[i][j].w};
#pragma unroll
                        for (int h = 0; h < 2; ++h) {
                            const int v = v0 + i * 16 + gid + 8 * h;
                            if (v < dim) o[v] = acc[i][j][2 * h + x] + y[2 * h + x];
                        }
                    }
                }
        }
    }
    if (carries) {
        float* dst = cm.state + ((int64_t)sl.out * cm.heads + head) * dim * KD;
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int v = v0 + i * 16 + gid + 8 * h;
                    if (v < dim) *reinterpret_cast<float2*>(dst + (int64_t)v * KD + tile * 16 + j * 8 + 2 * tq) = make_float2(S[i][j][2 * h], S[i][j][2 * h + 1]);
                }
    }
}

template <int KD>
void launch_chunks(const ChannelDeltaArgs& a, int longest, void* scratch, cudaStream_t s) {
    const LinearStateArgs& c = a.common;
    auto* chunk = channel_delta_chunk_kernel<KD>;
    auto* states = channel_delta_states_kernel<KD>;
    ensure_dynamic_smem(reinterpret_cast<const void*>(chunk), ChunkSmem<KD>::BYTES);
    ensure_dynamic_smem(reinterpret_cast<const void*>(states), StatesSmem<KD>::BYTES);
    bool vec = a.y.ld % 4 == 0 && a.y.stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a.y.p) & 15) == 0 && c.dim % 4 == 0;
    for (int col : {a.r_col, a.k_col, a.v_col, a.a_col}) vec = vec && col % 4 == 0;
    const int chunks = (longest + CC_ROWS - 1) / CC_ROWS;
    uint8_t* results = static_cast<uint8_t*>(scratch);
    launch_pdl(chunk, dim3((unsigned)c.heads, (unsigned)chunks, (unsigned)c.lanes.lanes), dim3(CC_THREADS), ChunkSmem<KD>::BYTES, s, a, results, vec ? 1 : 0);
    MK_LAUNCH_CHECK();
    launch_pdl(states, dim3((unsigned)((c.dim + CC_SLICE - 1) / CC_SLICE), (unsigned)c.heads, (unsigned)c.lanes.lanes), dim3(StatesSmem<KD>::WARPS * 32),
               StatesSmem<KD>::BYTES, s, a, static_cast<const uint8_t*>(results));
    MK_LAUNCH_CHECK();
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

bool channel_delta_can_chunk(int dim) { return dim > 32 && dim <= 128; }

size_t channel_delta_chunk_bytes(int dim, int heads, int tokens, int lanes) {
    if (!channel_delta_can_chunk(dim)) return 0;
    const size_t one = linear_state_key_pad(dim) == 64 ? ChunkResult<64>::BYTES : ChunkResult<128>::BYTES;
    return ((size_t)tokens / CC_ROWS + (size_t)lanes + 1) * (size_t)heads * one;
}

void launch_channel_delta_chunks(const ChannelDeltaArgs& a, int longest, void* scratch, cudaStream_t s) {
    if (a.common.lanes.lanes <= 0 || longest <= 0) return;
    if (!channel_delta_can_chunk(a.common.dim) || a.common.dim != a.common.vdim || a.w2h == nullptr)
        throw std::runtime_error("delta-rule chunks with channel gates: square heads of 33 to 128, a bfloat16 low-rank matrix");
    if (a.common.lanes.lanes > 65535 || a.common.heads > 65535 || longest > 65535 * CC_ROWS) throw std::runtime_error("delta-rule chunks with channel gates: too many lanes, heads or rows");
    if (linear_state_key_pad(a.common.dim) == 64) launch_chunks<64>(a, longest, scratch, s);
    else launch_chunks<128>(a, longest, scratch, s);
}

}  // namespace mk
