// The matrix memory of mLSTM (see MlstmScanArgs): one-token lanes and prompts.  State layout as in linear_state.h; the last column
// is the normaliser.
//
// mlstm_step_kernel: ticks of one-token lanes.  A warp holds 2048 numbers of the state (whole columns) in registers, requested before
// the predecessor is waited for; the CTA that arrives last at a head's counter norms and gates the head's row.
//
// mlstm_chunk_kernel: prompts, 64 rows at a time, tensor cores.  With F the running sum of the log forget gates of a chunk, m_t the
// running maximum and m_0, S, n what the chunk starts from,
//   c_s = i_s - F_s,  e_t = m_t - F_t:   D_ts = exp(c_s - e_t) (s <= t),  g_t = exp(m_0 - e_t),
//   o_t = sum_s D_ts (q_t . k_s) v_s + g_t S^T q_t,   S' = g_last S + sum_s exp(c_s - e_last) k_s v_s^T,
// every exponent at most 0.  q, k and v are bfloat16 numbers, as the projection's epilogue leaves them; what the recurrence adds to them - D (Q K^T), the written values and the
// state - enters a product as the sum of two bfloat16 numbers (16 bits and more), and the state itself stays in f32 registers.
#include "linear_state.h"
#include "device_util.h"
#include "mma_bf16.cuh"
#include "recurrent_core.cuh"
#include <algorithm>

namespace mk {

namespace {

// The logarithms of a row's input and forget gate.
__device__ __forceinline__ float log_input_gate(const MlstmScanArgs& a, int64_t row, int head) {
    return a.cap * tanhf((a.y.at(row, a.i_col + head) + a.i_bias[head]) / a.cap);
}
__device__ __forceinline__ float log_forget_gate(const MlstmScanArgs& a, int64_t row, int head) {
    return -recurrent::softplus_stable(-a.cap * tanhf((a.y.at(row, a.f_col + head) + a.f_bias[head]) / a.cap));
}

// ------------------------------------------------------------------------------------------------ one-token lanes

constexpr int MS_WARPS = 4;

template <int KD>
struct Step {
    static constexpr int LPC = KD >= 128 ? 32 : KD / 4;  // lanes of a column, four keys each
    static constexpr int CPW = 32 / LPC;                 // columns a warp loads at once
    static constexpr int NJ = KD / (4 * LPC);            // four-key packs of a lane and column
    static constexpr int SLOTS = 16 / NJ;                // columns of a lane
    static constexpr int WARP_COLS = SLOTS * CPW;
    static constexpr int COLS = MS_WARPS * WARP_COLS;    // columns of a CTA
};

template <int KD>
__global__ void __launch_bounds__(MS_WARPS * 32, 4) mlstm_step_kernel(const __grid_constant__ MlstmScanArgs a, int vec) {
    using P = Step<KD>;
    constexpr int LPC = P::LPC, CPW = P::CPW, NJ = P::NJ, SLOTS = P::SLOTS;
    __shared__ float s_v[P::COLS], s_o[P::COLS], red[MS_WARPS], s_den;
    __shared__ int s_last;
    const LinearStateArgs& c = a.common;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lk = lane & (LPC - 1), lc = lane / LPC;
    const int unit = blockIdx.x, head = blockIdx.y, col0 = unit * P::COLS, w0 = warp * P::WARP_COLS;
    const int64_t head_state = (int64_t)(c.vdim + 1) * KD;

    pdl_trigger();
    const StateLane sl = c.lanes.at(blockIdx.z);
    float4 S[SLOTS][NJ], n[NJ];
    const float4* src = reinterpret_cast<const float4*>(c.state + ((int64_t)sl.in * c.heads + head) * head_state);
#pragma unroll
    for (int s = 0; s < SLOTS; ++s) {
        const int col = col0 + w0 + s * CPW + lc;
        const bool live = sl.in >= 0 && col < c.vdim;
#pragma unroll
        for (int j = 0; j < NJ; ++j) S[s][j] = live ? __ldcs(src + (int64_t)col * (KD / 4) + j * LPC + lk) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < NJ; ++j)
        n[j] = sl.in >= 0 && warp == 0 && lc == 0 ? __ldcg(src + (int64_t)c.vdim * (KD / 4) + j * LPC + lk) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float before = sl.in >= 0 ? a.running_max[(int64_t)sl.in * c.heads + head] : 0.f;
    pdl_wait();

    const int64_t row = sl.first;
    float4 q[NJ], k[NJ];
    // the numbers a prompt's chunks would multiply
    auto operand = [&](float x) { return a.rounded ? __bfloat162float(__float2bfloat16_rn(x)) : x; };
    auto keys = [&](int col, int j) {
        const int d = (j * LPC + lk) * 4;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (vec) {
            if (d < c.dim) x = a.y.at4(row, col + d);
        } else {
            if (d < c.dim) x.x = a.y.at(row, col + d);
            if (d + 1 < c.dim) x.y = a.y.at(row, col + d + 1);
            if (d + 2 < c.dim) x.z = a.y.at(row, col + d + 2);
            if (d + 3 < c.dim) x.w = a.y.at(row, col + d + 3);
        }
        return make_float4(operand(x.x), operand(x.y), operand(x.z), operand(x.w));
    };
    for (int i = threadIdx.x; i < P::COLS; i += MS_WARPS * 32)
        s_v[i] = col0 + i < c.vdim ? operand(a.y.at(row, a.v_col + head * c.vdim + col0 + i)) : 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        q[j] = keys(a.q_col + head * c.dim, j);
        k[j] = keys(a.k_col + head * c.dim, j);
    }
    const float li = log_input_gate(a, row, head), lf = log_forget_gate(a, row, head);
    const float top = fmaxf(lf + before, li), keep = expf(lf + before - top), write = expf(li - top), q_scale = rsqrtf((float)c.dim);
    __syncthreads();

    float part[SLOTS];
    float4* dst = reinterpret_cast<float4*>(c.state + ((int64_t)sl.out * c.heads + head) * head_state);
#pragma unroll
    for (int s = 0; s < SLOTS; ++s) {
        const int at = w0 + s * CPW + lc;
        const float u = write * s_v[at];
        part[s] = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            float4 x = S[s][j];
            x.x = fmaf(k[j].x, u, keep * x.x);
            x.y = fmaf(k[j].y, u, keep * x.y);
            x.z = fmaf(k[j].z, u, keep * x.z);
            x.w = fmaf(k[j].w, u, keep * x.w);
            part[s] = fmaf(x.x, q[j].x, fmaf(x.y, q[j].y, fmaf(x.z, q[j].z, fmaf(x.w, q[j].w, part[s]))));
            if (col0 + at < c.vdim) __stcs(dst + (int64_t)(col0 + at) * (KD / 4) + j * LPC + lk, x);
        }
    }
    int first;
    const int held = fold_lanes<SLOTS, LPC>(part, lane, first);
#pragma unroll
    for (int i = 0; i < SLOTS; ++i)
        if (i < held) s_o[w0 + (first + i) * CPW + lc] = part[i] * q_scale;  // lanes that share a column write the same number
    if (warp == 0) {
        float nq = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            float4 x = n[j];
            x.x = fmaf(k[j].x, write, keep * x.x);
            x.y = fmaf(k[j].y, write, keep * x.y);
            x.z = fmaf(k[j].z, write, keep * x.z);
            x.w = fmaf(k[j].w, write, keep * x.w);
            nq = fmaf(x.x, q[j].x, fmaf(x.y, q[j].y, fmaf(x.z, q[j].z, fmaf(x.w, q[j].w, nq))));
            if (unit == 0 && lc == 0) __stcs(dst + (int64_t)c.vdim * (KD / 4) + j * LPC + lk, x);
        }
#pragma unroll
        for (int x = 1; x < LPC; x <<= 1) nq += __shfl_xor_sync(0xffffffffu, nq, x);
        if (lane == 0) {
            s_den = fmaxf(fabsf(nq * q_scale), expf(-top)) + 1e-6f;
            if (unit == 0) a.running_max[(int64_t)sl.out * c.heads + head] = top;
        }
    }
    __syncthreads();

    // the head's row: from here when one CTA holds it, otherwise by way of memory in the CTA that comes last
    const bool alone = gridDim.x == 1;
    float* raw = c.out + ((int64_t)row * c.heads + head) * linear_state_raw_width(c.vdim);
    if (!alone) {
        for (int i = threadIdx.x; i < P::COLS && col0 + i < c.vdim; i += MS_WARPS * 32) raw[col0 + i] = s_o[i] / s_den;
        __threadfence();
        __syncthreads();
        if (threadIdx.x == 0) {
            int32_t* counter = a.counters + (int64_t)blockIdx.z * c.heads + head;
            s_last = atomicAdd(counter, 1) == (int)gridDim.x - 1;
            if (s_last) *counter = 0;
        }
        __syncthreads();
        if (!s_last) return;
        __threadfence();
    }
    auto value = [&](int v) { return alone ? s_o[v] / s_den : __ldcg(raw + v); };
    float ss = 0.f;
    for (int v = threadIdx.x; v < c.vdim; v += MS_WARPS * 32) ss = fmaf(value(v), value(v), ss);
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = red[0];
#pragma unroll
    for (int w = 1; w < MS_WARPS; ++w) ss += red[w];
    const float root = sqrtf(ss / (float)c.vdim + c.eps);
    const float* nw = c.norm_w + (c.norm_per_head ? head * c.vdim : 0);
    for (int v = threadIdx.x; v < c.vdim; v += MS_WARPS * 32) {
        const float g = c.gate.at(row, c.gate_col + head * c.vdim + v);
        c.image.put(row, head * c.vdim + v, value(v) / root * nw[v] * (c.gate_sigmoid ? sigmoid_f(g) : silu_f(g)));
    }
    if (head == c.heads - 1)
        for (int x = c.heads * c.vdim + threadIdx.x; x < c.image.end(); x += MS_WARPS * 32) c.image.put(row, x, 0.f);
}

// ------------------------------------------------------------------------------------------------ prompts

constexpr int MC_ROWS = 64;      // rows of a chunk
constexpr int MC_WARPS = 16;
constexpr int MC_THREADS = MC_WARPS * 32;           // that compute; one more warp keeps the gates a chunk ahead

// All warps of the CTA, the gates' one included.
__device__ __forceinline__ void mc_sync() { asm volatile("bar.sync 1, %0;" ::"n"(MC_THREADS + 32) : "memory"); }

// acc[N] (16 rows x 8 N columns) += A B over 16 STEPS inner indices, B in one or two parts.
//   a_at(step): fragment of A.  b_at(step, tile): where the tile's 16 inner indices begin, its columns (or, TRANS, its inner indices)
//   PITCH apart.
// Pairs of tiles share a load; a single tile takes two steps per load.
template <int N, int STEPS, bool TRANS, int PITCH, typename A, typename B>
__device__ __forceinline__ void mc_product(float (&acc)[N][4], int lane, A a_at, B b_at, const __nv_bfloat16* b_hi, const __nv_bfloat16* b_lo) {
    // lane's row of the four 8 x 8 matrices of a load
    const int pair = TRANS ? ((lane & 7) + ((lane >> 3) & 1) * 8) * PITCH + (lane >> 4) * 8 : ((lane & 7) + (lane >> 4) * 8) * PITCH + ((lane >> 3) & 1) * 8;
    const int single = TRANS ? lane * PITCH : (lane & 7) * PITCH + (lane >> 3) * 8;
    auto load = [&](uint32_t (&r)[4], const __nv_bfloat16* p) {
        if (TRANS) mc_ldmatrix_t(r, p);
        else mc_ldmatrix(r, p);
    };
    if constexpr (N % 2 == 0) {
#pragma unroll
        for (int k = 0; k < STEPS; ++k) {
            uint32_t af[4], bf[4];
            a_at(k, af);
#pragma unroll
            for (int j = 0; j < N; j += 2) {
                load(bf, b_hi + b_at(k, j) + pair);
                mc_mma(acc[j], af, bf[0], bf[1]);
                mc_mma(acc[j + 1], af, bf[2], bf[3]);
                if (b_lo != nullptr) {
                    load(bf, b_lo + b_at(k, j) + pair);
                    mc_mma(acc[j], af, bf[0], bf[1]);
                    mc_mma(acc[j + 1], af, bf[2], bf[3]);
                }
            }
        }
    } else {
        static_assert(N == 1 && STEPS % 2 == 0, "a single tile takes pairs of steps");
#pragma unroll
        for (int k = 0; k < STEPS; k += 2) {
            uint32_t a0[4], a1[4], bf[4];
            a_at(k, a0);
            a_at(k + 1, a1);
            load(bf, b_hi + b_at(k, 0) + single);
            mc_mma(acc[0], a0, bf[0], bf[1]);
            mc_mma(acc[0], a1, bf[2], bf[3]);
            if (b_lo != nullptr) {
                load(bf, b_lo + b_at(k, 0) + single);
                mc_mma(acc[0], a0, bf[0], bf[1]);
                mc_mma(acc[0], a1, bf[2], bf[3]);
            }
        }
    }
}

template <int KD, int C>
struct Chunk {
    static constexpr int KP = KD + 8, CP = C + 8, PP = MC_ROWS + 8;  // padded rows (bfloat16): conflict-free ldmatrix
    static constexpr int COL_GROUPS = C / 16, KEY_GROUPS = MC_WARPS / COL_GROUPS, KEYS = KD / KEY_GROUPS;  // of the state, by warp
    static constexpr int N_PARTS = MC_THREADS / (KD / 2);            // row groups of the normaliser's sums
    static constexpr int INPUTS = MC_ROWS * (2 * KP + CP);           // one chunk's q, k, v
    static constexpr int HALVES = 2 * INPUTS + 2 * MC_ROWS * CP + 2 * MC_ROWS * PP + 2 * C * KP;
    static constexpr int GATES = 7 * MC_ROWS + 4;                    // one chunk's
    static constexpr int FLOATS = 2 * GATES + 5 * MC_ROWS + KD + N_PARTS * KD;
    static constexpr size_t BYTES = (size_t)HALVES * 2 + (size_t)FLOATS * 4;
    static_assert(KEYS % 8 == 0 && C % 32 == 0 && BYTES <= 227 * 1024, "whole tiles that fit");
};

// What the chunk's exponents are made of (see the top), by row.
struct ChunkGates {
    float2 *c, *e;                    // in units of ln 2, two parts each
    float *g, *w, *floor, *keep;
    __device__ __forceinline__ explicit ChunkGates(float* at) {
        c = reinterpret_cast<float2*>(at);
        e = c + MC_ROWS;
        g = reinterpret_cast<float*>(e + MC_ROWS);
        w = g + MC_ROWS;
        floor = w + MC_ROWS;
        keep = floor + MC_ROWS;
    }
};

// One warp, two rows per lane: the gates of `m` rows behind a running maximum, which it moves on.  Sums and maxima in f64:
// differences of far sums stay exact.
__device__ __forceinline__ void chunk_gates(const MlstmScanArgs& a, int64_t first, int m, int head, float& run_max, const ChunkGates& out, int lane) {
    constexpr double kLog2e = 1.4426950408889634074;
    double li[2], lf[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int r = 2 * lane + h;
        li[h] = r < m ? (double)log_input_gate(a, first + r, head) : -INFINITY;  // rows past the end change neither sums nor maxima
        lf[h] = r < m ? (double)log_forget_gate(a, first + r, head) : 0.0;
    }
    double f1 = lf[0] + lf[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double p = __shfl_up_sync(0xffffffffu, f1, o);
        if (lane >= o) f1 += p;
    }
    const double F[2] = {f1 - lf[1], f1};
    const double c[2] = {li[0] - F[0], li[1] - F[1]};
    double best = fmax(c[0], c[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double p = __shfl_up_sync(0xffffffffu, best, o);
        if (lane >= o) best = fmax(best, p);
    }
    double earlier = __shfl_up_sync(0xffffffffu, best, 1);
    if (lane == 0) earlier = -INFINITY;
    const double top[2] = {F[0] + fmax((double)run_max, fmax(earlier, c[0])), F[1] + fmax((double)run_max, best)};
    double e[2];
    float mt[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        mt[h] = (float)top[h];
        e[h] = (double)mt[h] - F[h];
    }
    const double e_last = __shfl_sync(0xffffffffu, e[1], 31);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int r = 2 * lane + h;
        const double c2 = c[h] * kLog2e, e2 = e[h] * kLog2e;
        const float c_hi = (float)c2, e_hi = (float)e2;
        out.c[r] = make_float2(c_hi, r < m ? (float)(c2 - (double)c_hi) : 0.f);
        out.e[r] = make_float2(e_hi, (float)(e2 - (double)e_hi));
        out.g[r] = expf((float)(run_max - e[h]));
        out.w[r] = expf((float)(c[h] - e_last));
        out.floor[r] = expf(-mt[h]);
    }
    if (lane == 0) *out.keep = expf((float)(run_max - e_last));
    run_max = __shfl_sync(0xffffffffu, mt[1], 31);
}

// Grid (column slices of C, heads, lanes).  vec: rows of q, k and v in whole 16-byte pieces.
template <int KD, int C>
__global__ void __launch_bounds__(MC_THREADS + 32, 1) mlstm_chunk_kernel(const __grid_constant__ MlstmScanArgs a, int vec) {
    using P = Chunk<KD, C>;
    constexpr int KP = P::KP, CP = P::CP, PP = P::PP, R = MC_ROWS;
    constexpr int NT = C / 32;            // output tiles of a warp: 16 rows x C / 4 columns
    constexpr int NK = P::KEYS / 8;       // state tiles of a warp: 16 columns x KEYS keys
    extern __shared__ __align__(16) unsigned char mc_raw[];
    __nv_bfloat16* inputs = reinterpret_cast<__nv_bfloat16*>(mc_raw);  // [2]: q [R][KP], k [R][KP], v [R][CP]
    __nv_bfloat16* Wh = inputs + 2 * P::INPUTS;                     // written values, [R][CP] in two parts
    __nv_bfloat16* Wl = Wh + R * CP;
    __nv_bfloat16* Ph = Wl + R * CP;                                // D (Q K^T), [R][PP] in two parts
    __nv_bfloat16* Pl = Ph + R * PP;
    __nv_bfloat16* Sh = Pl + R * PP;                                // the state the chunk starts from, [C][KP] in two parts
    __nv_bfloat16* Sl = Sh + C * KP;
    float* gates = reinterpret_cast<float*>(Sl + C * KP);           // [2]
    float *s_nq = gates + 2 * P::GATES, *s_sum = s_nq + R /* [4][R] */, *s_n = s_sum + 4 * R, *s_np = s_n + KD /* [N_PARTS][KD] */;

    const LinearStateArgs& cm = a.common;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tq = lane & 3;
    const int col0 = blockIdx.x * C, head = blockIdx.y, cols = min(C, cm.vdim - col0);
    const int64_t head_state = (int64_t)(cm.vdim + 1) * KD;
    const int sc0 = warp % P::COL_GROUPS * 16, sk0 = warp / P::COL_GROUPS * P::KEYS;  // the warp's part of the state
    const int row0 = (warp & 3) * 16, quarter = warp >> 2;                            // its part of a chunk's rows

    pdl_trigger();
    const StateLane sl = cm.lanes.at(blockIdx.z);
    const int n = sl.n, chunks = (n + R - 1) / R;

    if (warp == MC_WARPS) {
        // the gates' warp: a chunk ahead of the others, whom it meets at every barrier
        float run_max = sl.in >= 0 ? a.running_max[(int64_t)sl.in * cm.heads + head] : 0.f;
        pdl_wait();
        for (int ch = 0; ch <= chunks; ++ch) {
            if (ch < chunks) chunk_gates(a, sl.first + (int64_t)ch * R, min(R, n - ch * R), head, run_max, ChunkGates(gates + (ch & 1) * P::GATES), lane);
            if (ch > 0) {
                mc_sync();
                mc_sync();
            }
            if (ch < chunks) mc_sync();
        }
        if (blockIdx.x == 0 && lane == 0) a.running_max[(int64_t)sl.out * cm.heads + head] = run_max;
        return;
    }

    float S[NK][4];
    {
        const float* src = cm.state + ((int64_t)sl.in * cm.heads + head) * head_state;
#pragma unroll
        for (int j = 0; j < NK; ++j)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int col = col0 + sc0 + gid + 8 * h;
                float2 x = make_float2(0.f, 0.f);
                if (sl.in >= 0 && col < cm.vdim) x = *reinterpret_cast<const float2*>(src + (int64_t)col * KD + sk0 + j * 8 + 2 * tq);
                S[j][2 * h] = x.x;
                S[j][2 * h + 1] = x.y;
            }
        for (int i = threadIdx.x; i < KD; i += MC_THREADS) s_n[i] = sl.in >= 0 ? src[(int64_t)cm.vdim * KD + i] : 0.f;
    }
    auto publish_state = [&] {
#pragma unroll
        for (int j = 0; j < NK; ++j)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                uint32_t hi, lo;
                mc_split(S[j][2 * h], S[j][2 * h + 1], hi, lo);
                const int at = (sc0 + gid + 8 * h) * KP + sk0 + j * 8 + 2 * tq;
                *reinterpret_cast<uint32_t*>(Sh + at) = hi;
                *reinterpret_cast<uint32_t*>(Sl + at) = lo;
            }
    };
    publish_state();
    pdl_wait();

    const int qc = a.q_col + head * cm.dim, kc = a.k_col + head * cm.dim, vc = a.v_col + head * cm.vdim + col0;
    // a chunk's q, k and v on their way; rows past the end and columns past the head are zeros
    auto request = [&](int chunk) {
        __nv_bfloat16* Q = inputs + (chunk & 1) * P::INPUTS;
        __nv_bfloat16 *K = Q + R * KP, *V = K + R * KP;
        const __nv_bfloat16* y = a.yh + ((int64_t)sl.first + (int64_t)chunk * R) * a.ldh;
        const int m = min(R, n - chunk * R);
        if (vec) {
#pragma unroll
            for (int i = threadIdx.x; i < R * (KD / 8); i += MC_THREADS) {
                const int r = i / (KD / 8), c = i % (KD / 8) * 8;
                const bool live = r < m && c < cm.dim;
                const __nv_bfloat16* src = y + (live ? (int64_t)r * a.ldh + c : 0);
                mc_cp_async16(Q + r * KP + c, src + qc, live);
                mc_cp_async16(K + r * KP + c, src + kc, live);
            }
            for (int i = threadIdx.x; i < R * (C / 8); i += MC_THREADS) {
                const int r = i / (C / 8), c = i % (C / 8) * 8;
                const bool live = r < m && c < cols;
                mc_cp_async16(V + r * CP + c, y + vc + (live ? (int64_t)r * a.ldh + c : 0), live);
            }
        } else {
            const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);
            for (int i = threadIdx.x; i < R * KD; i += MC_THREADS) {
                const int r = i / KD, c = i % KD;
                const bool live = r < m && c < cm.dim;
                Q[r * KP + c] = live ? y[(int64_t)r * a.ldh + qc + c] : zero;
                K[r * KP + c] = live ? y[(int64_t)r * a.ldh + kc + c] : zero;
            }
            for (int i = threadIdx.x; i < R * C; i += MC_THREADS) {
                const int r = i / C, c = i % C;
                V[r * CP + c] = r < m && c < cols ? y[(int64_t)r * a.ldh + vc + c] : zero;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (chunks > 0) request(0);
    const float q_scale = rsqrtf((float)cm.dim);
    const bool even = (cm.vdim & 1) == 0;

    for (int ch = 0; ch < chunks; ++ch) {
        const int64_t r0 = sl.first + (int64_t)ch * R;
        const int m = min(R, n - ch * R);
        const ChunkGates gt(gates + (ch & 1) * P::GATES);
        const __nv_bfloat16* Q = inputs + (ch & 1) * P::INPUTS;
        const __nv_bfloat16 *K = Q + R * KP, *V = K + R * KP;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        mc_sync();  // the chunk's inputs and gates, the state and the normaliser it starts from
        if (ch + 1 < chunks) request(ch + 1);
        // what the rows write: v times the weight that is left of it at the chunk's end
#pragma unroll
        for (int i = threadIdx.x; i < R * (C / 2); i += MC_THREADS) {
            const int r = i / (C / 2), c = i % (C / 2) * 2;
            const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(V + r * CP + c);
            uint32_t hi, lo;
            mc_split(gt.w[r] * __low2float(v), gt.w[r] * __high2float(v), hi, lo);
            *reinterpret_cast<uint32_t*>(Wh + r * CP + c) = hi;
            *reinterpret_cast<uint32_t*>(Wl + r * CP + c) = lo;
        }
        auto q_fragment = [&](int k, uint32_t (&r)[4]) { mc_ldmatrix(r, Q + (row0 + (lane & 15)) * KP + k * 16 + (lane >> 4) * 8); };

        // D (Q K^T): 16 rows x 16 keys per warp, keys behind the rows are zeros
        {
            float sc[2][4] = {}, sum[2] = {0.f, 0.f};
            const int k0 = quarter * 16;
            uint32_t hi[2][2] = {}, lo[2][2] = {};
            if (k0 <= row0) {
                mc_product<2, KD / 16, false, KP>(sc, lane, q_fragment, [&](int k, int j) { return (k0 + j * 8) * KP + k * 16; }, K, nullptr);
                const float2 e[2] = {gt.e[row0 + gid], gt.e[row0 + gid + 8]};
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int s = k0 + j * 8 + 2 * tq;
                    const float4 c = *reinterpret_cast<const float4*>(gt.c + s);
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
                        const int t = row0 + gid + 8 * h;
                        const float d0 = s <= t ? exp2f((c.x - e[h].x) + (c.y - e[h].y)) : 0.f, d1 = s + 1 <= t ? exp2f((c.z - e[h].x) + (c.w - e[h].y)) : 0.f;
                        const float p0 = sc[j][2 * h] * q_scale * d0, p1 = sc[j][2 * h + 1] * q_scale * d1;
                        sum[h] += p0 + p1;
                        mc_split(p0, p1, hi[j][h], lo[j][h]);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int at = (row0 + gid + 8 * h) * PP + k0 + j * 8 + 2 * tq;
                    *reinterpret_cast<uint32_t*>(Ph + at) = hi[j][h];
                    *reinterpret_cast<uint32_t*>(Pl + at) = lo[j][h];
                }
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 1);
                sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 2);
                if (tq == 0) s_sum[quarter * R + row0 + gid + 8 * h] = sum[h];
            }
            // n . q of the normaliser the chunk starts from: eight threads per row
            const int t = threadIdx.x >> 3, part = threadIdx.x & 7;
            float nq = 0.f;
#pragma unroll
            for (int c = part * 2; c < KD; c += 16) {
                const __nv_bfloat162 q2 = *reinterpret_cast<const __nv_bfloat162*>(Q + t * KP + c);
                const float2 n2 = *reinterpret_cast<const float2*>(s_n + c);
                nq = fmaf(__low2float(q2), n2.x, fmaf(__high2float(q2), n2.y, nq));
            }
#pragma unroll
            for (int x = 1; x < 8; x <<= 1) nq += __shfl_xor_sync(0xffffffffu, nq, x);
            if (part == 0) s_nq[t] = nq;
        }
        mc_sync();

        // outputs: 16 rows x C / 4 columns per warp
        {
            float o[NT][4] = {};
            const int n0 = quarter * (C / 4);
            mc_product<NT, KD / 16, false, KP>(o, lane, q_fragment, [&](int k, int j) { return (n0 + j * 8) * KP + k * 16; }, Sh, Sl);
            float g[2], den[2];
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int t = row0 + gid + 8 * h;
                g[h] = gt.g[t] * q_scale;
                const float nq = s_sum[t] + s_sum[R + t] + s_sum[2 * R + t] + s_sum[3 * R + t] + g[h] * s_nq[t];
                den[h] = fmaxf(fabsf(nq), gt.floor[t]) + 1e-6f;
            }
#pragma unroll
            for (int j = 0; j < NT; ++j)
#pragma unroll
                for (int x = 0; x < 4; ++x) o[j][x] *= g[x >> 1];
            // the weights behind the rows are zeros: only what lies before counts, 32 keys at a time
            auto v_at = [&](int k, int j) { return k * 16 * CP + n0 + j * 8; };
#pragma unroll
            for (int part = 0; part < 2; ++part) {
                const __nv_bfloat16* Pp = part == 0 ? Ph : Pl;
                auto p_fragment = [&](int k, uint32_t (&r)[4]) { mc_ldmatrix(r, Pp + (row0 + (lane & 15)) * PP + k * 16 + (lane >> 4) * 8); };
                if (row0 < 32) mc_product<NT, 2, true, CP>(o, lane, p_fragment, v_at, V, nullptr);
                else mc_product<NT, 4, true, CP>(o, lane, p_fragment, v_at, V, nullptr);
            }
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int t = row0 + gid + 8 * h;
                if (t >= m) continue;
                float* out = cm.out + ((r0 + t) * cm.heads + head) * cm.vdim + col0;
                const float inv = 1.0f / den[h];
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    const int c = n0 + j * 8 + 2 * tq;
                    const float x = o[j][2 * h] * inv, y = o[j][2 * h + 1] * inv;
                    if (even) {
                        if (c < cols) *reinterpret_cast<float2*>(out + c) = make_float2(x, y);
                    } else {
                        if (c < cols) out[c] = x;
                        if (c + 1 < cols) out[c + 1] = y;
                    }
                }
            }
        }
        // the state behind the chunk: 16 columns x KEYS keys per warp
        const float keep = *gt.keep;
#pragma unroll
        for (int j = 0; j < NK; ++j)
#pragma unroll
            for (int x = 0; x < 4; ++x) S[j][x] *= keep;
        auto k_at = [&](int k, int j) { return k * 16 * KP + sk0 + j * 8; };
#pragma unroll
        for (int part = 0; part < 2; ++part) {
            const __nv_bfloat16* Wp = part == 0 ? Wh : Wl;
            auto w_fragment = [&](int k, uint32_t (&r)[4]) { mc_ldmatrix_t(r, Wp + (k * 16 + (lane >> 4) * 8 + (lane & 7)) * CP + sc0 + ((lane >> 3) & 1) * 8); };
            mc_product<NK, R / 16, true, KP>(S, lane, w_fragment, k_at, K, nullptr);
        }
        {
            const int pair = threadIdx.x % (KD / 2) * 2, part = threadIdx.x / (KD / 2);
            constexpr int ROWS = R / P::N_PARTS;
            float x = 0.f, y = 0.f;
#pragma unroll
            for (int t = part * ROWS; t < (part + 1) * ROWS; ++t) {
                const __nv_bfloat162 k2 = *reinterpret_cast<const __nv_bfloat162*>(K + t * KP + pair);
                x = fmaf(gt.w[t], __low2float(k2), x);
                y = fmaf(gt.w[t], __high2float(k2), y);
            }
            *reinterpret_cast<float2*>(s_np + part * KD + pair) = make_float2(x, y);
        }
        mc_sync();  // the old state was read by everyone
        publish_state();
        for (int i = threadIdx.x; i < KD; i += MC_THREADS) {
            float x = s_n[i] * keep;
#pragma unroll
            for (int p = 0; p < P::N_PARTS; ++p) x += s_np[p * KD + i];
            s_n[i] = x;
        }
    }

    float* dst = cm.state + ((int64_t)sl.out * cm.heads + head) * head_state;
#pragma unroll
    for (int j = 0; j < NK; ++j)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int col = col0 + sc0 + gid + 8 * h;
            if (col < cm.vdim) *reinterpret_cast<float2*>(dst + (int64_t)col * KD + sk0 + j * 8 + 2 * tq) = make_float2(S[j][2 * h], S[j][2 * h + 1]);
        }
    if (blockIdx.x == 0) {
        for (int i = threadIdx.x; i < KD; i += MC_THREADS) dst[(int64_t)cm.vdim * KD + i] = s_n[i];  // written by the same thread
    }
}

bool aligned_heads(const MlstmScanArgs& a) {
    const LinearStateArgs& c = a.common;
    bool ok = a.y.ld % 4 == 0 && a.y.stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a.y.p) & 15) == 0 && c.dim % 4 == 0 && c.vdim % 4 == 0;
    for (int col : {a.q_col, a.k_col, a.v_col}) ok = ok && col % 4 == 0;
    return ok;
}

template <int KD>
void launch_step(const MlstmScanArgs& a, cudaStream_t s) {
    const LinearStateArgs& c = a.common;
    const dim3 grid((unsigned)((c.vdim + Step<KD>::COLS - 1) / Step<KD>::COLS), (unsigned)c.heads, (unsigned)c.lanes.lanes);
    if (grid.x > 1 && a.counters == nullptr) throw std::runtime_error("mLSTM step: counters are missing");
    launch_pdl(mlstm_step_kernel<KD>, grid, dim3(MS_WARPS * 32), 0, s, a, aligned_heads(a) ? 1 : 0);
    MK_LAUNCH_CHECK();
}

template <int KD, int C>
void launch_chunk_cols(const MlstmScanArgs& a, cudaStream_t s) {
    const LinearStateArgs& c = a.common;
    auto* kernel = mlstm_chunk_kernel<KD, C>;
    ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), Chunk<KD, C>::BYTES);
    const bool vec = a.ldh % 8 == 0 && c.dim % 8 == 0 && c.vdim % 8 == 0 && a.q_col % 8 == 0 && a.k_col % 8 == 0 && a.v_col % 8 == 0 &&
                     (reinterpret_cast<uintptr_t>(a.yh) & 15) == 0;
    const dim3 grid((unsigned)((c.vdim + C - 1) / C), (unsigned)c.heads, (unsigned)c.lanes.lanes);
    launch_pdl(kernel, grid, dim3(MC_THREADS + 32), Chunk<KD, C>::BYTES, s, a, vec ? 1 : 0);
    MK_LAUNCH_CHECK();
}

// Narrow column slices while they are what fills the GPU: every slice repeats Q K^T.
template <int KD>
void launch_chunk(const MlstmScanArgs& a, cudaStream_t s) {
    const LinearStateArgs& c = a.common;
    if ((int64_t)(c.vdim + 63) / 64 * c.heads * c.lanes.lanes >= device_sm_count()) launch_chunk_cols<KD, 64>(a, s);
    else launch_chunk_cols<KD, 32>(a, s);
}

}  // namespace

void launch_mlstm_step(const MlstmScanArgs& a, cudaStream_t s) {
    switch (linear_state_key_pad(a.common.dim)) {
        case 32: launch_step<32>(a, s); break;
        case 64: launch_step<64>(a, s); break;
        case 128: launch_step<128>(a, s); break;
        default: launch_step<256>(a, s); break;
    }
}

void launch_mlstm_chunks(const MlstmScanArgs& a, cudaStream_t s) {
    switch (linear_state_key_pad(a.common.dim)) {
        case 32: launch_chunk_cols<32, 64>(a, s); break;
        case 64: launch_chunk<64>(a, s); break;
        case 128: launch_chunk<128>(a, s); break;
        default: launch_chunk_cols<256, 32>(a, s); break;
    }
}

}  // namespace mk
