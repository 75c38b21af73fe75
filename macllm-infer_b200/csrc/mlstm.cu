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
// every exponent at most 0.  q, k and v are bfloat16 numbers; what the recurrence adds to them - D (Q K^T), the written values and the
// state - enters a product as the sum of two bfloat16 numbers (16 bits and more), and the state itself stays in f32 registers.
#include "linear_state.h"
#include "device_util.h"
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
    auto operand = [&](float x) { return a.tensor_cores ? __bfloat162float(__float2bfloat16_rn(x)) : x; };
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
constexpr int MC_WARPS = 8;
constexpr int MC_THREADS = MC_WARPS * 32;

__device__ __forceinline__ uint32_t mc_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mc_ldmatrix(uint32_t (&r)[4], const __nv_bfloat16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mc_smem(p)));
}
__device__ __forceinline__ void mc_ldmatrix_t(uint32_t (&r)[4], const __nv_bfloat16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mc_smem(p)));
}
__device__ __forceinline__ void mc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mc_cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(mc_smem(dst)), "l"(src) : "memory");
}
// x and y as bfloat16 numbers, and what that left of them.
__device__ __forceinline__ void mc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

template <int KD, int C>
struct Chunk {
    static constexpr int KP = KD + 8, CP = C + 8, PP = MC_ROWS + 8;  // padded rows (bfloat16): conflict-free ldmatrix
    static constexpr int COL_GROUPS = C / 16, KEY_GROUPS = MC_WARPS / COL_GROUPS, KEYS = KD / KEY_GROUPS;  // of the state, by warp
    static constexpr bool STAGED = KD <= 128;                        // the next chunk's projections are on their way meanwhile
    static constexpr int HALVES = 2 * MC_ROWS * KP + 3 * MC_ROWS * CP + 2 * MC_ROWS * PP + 2 * C * KP;
    static constexpr int FLOATS = 11 * MC_ROWS + KD + 4;
    static constexpr int STAGE = STAGED ? MC_ROWS * (2 * KD + C) : 0;
    static constexpr size_t BYTES = (size_t)HALVES * 2 + (size_t)(FLOATS + STAGE) * 4;
    static_assert(KEYS % 16 == 0, "a warp takes pairs of key tiles");
};

// Grid (column slices of C, heads, lanes).
template <int KD, int C>
__global__ void __launch_bounds__(MC_THREADS, 1) mlstm_chunk_kernel(const __grid_constant__ MlstmScanArgs a, int vec) {
    using P = Chunk<KD, C>;
    constexpr int KP = P::KP, CP = P::CP, PP = P::PP, R = MC_ROWS;
    constexpr int NT = C / 16;            // output tiles of a warp: 16 rows x C / 2 columns
    constexpr int NK = P::KEYS / 8;       // state tiles of a warp: 16 columns x KEYS keys
    extern __shared__ __align__(16) unsigned char mc_raw[];
    __nv_bfloat16* Q = reinterpret_cast<__nv_bfloat16*>(mc_raw);   // [R][KP]
    __nv_bfloat16* K = Q + R * KP;                                  // [R][KP]
    __nv_bfloat16* V = K + R * KP;                                  // [R][CP]
    __nv_bfloat16* Wh = V + R * CP;                                 // written values, [R][CP] in two parts
    __nv_bfloat16* Wl = Wh + R * CP;
    __nv_bfloat16* Ph = Wl + R * CP;                                // D (Q K^T), [R][PP] in two parts
    __nv_bfloat16* Pl = Ph + R * PP;
    __nv_bfloat16* Sh = Pl + R * PP;                                // the state the chunk starts from, [C][KP] in two parts
    __nv_bfloat16* Sl = Sh + C * KP;
    float* c_hi = reinterpret_cast<float*>(Sl + C * KP);            // c_s and e_t in two parts each
    float *c_lo = c_hi + R, *e_hi = c_lo + R, *e_lo = e_hi + R, *s_g = e_lo + R, *s_w = s_g + R, *s_floor = s_w + R;
    float *s_sum = s_floor + R /* [2][R] */, *s_nq = s_sum + 2 * R, *s_n = s_nq + R + R /* spare */, *s_keep = s_n + KD;
    float* stage = s_keep + 4;                                      // [R][KD], [R][KD], [R][C]

    const LinearStateArgs& cm = a.common;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tq = lane & 3;
    const int col0 = blockIdx.x * C, head = blockIdx.y, cols = min(C, cm.vdim - col0);
    const int64_t head_state = (int64_t)(cm.vdim + 1) * KD;
    const int sc0 = warp % P::COL_GROUPS * 16, sk0 = warp / P::COL_GROUPS * P::KEYS;  // the warp's part of the state
    const int row0 = (warp & 3) * 16, half = warp >> 2;                               // its part of a chunk's rows

    pdl_trigger();
    const StateLane sl = cm.lanes.at(blockIdx.z);
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
    float run_max = sl.in >= 0 ? a.running_max[(int64_t)sl.in * cm.heads + head] : 0.f;  // warp 0's counts
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

    const int n = sl.n, chunks = (n + R - 1) / R;
    const int qc = a.q_col + head * cm.dim, kc = a.k_col + head * cm.dim, vc = a.v_col + head * cm.vdim + col0;
    const bool staged = P::STAGED && vec;
    float *st_q = stage, *st_k = stage + R * KD, *st_v = stage + 2 * R * KD;
    auto request = [&](int chunk) {
        const int64_t r0 = sl.first + (int64_t)chunk * R;
        const int m = min(R, n - chunk * R), kp = cm.dim >> 2, vp = cols >> 2;
        for (int i = threadIdx.x; i < m * kp; i += MC_THREADS) {
            const int r = i / kp, c = (i - r * kp) * 4;
            mc_cp_async16(st_q + r * KD + c, a.y.p + (r0 + r) * a.y.ld + qc + c);
            mc_cp_async16(st_k + r * KD + c, a.y.p + (r0 + r) * a.y.ld + kc + c);
        }
        for (int i = threadIdx.x; i < m * vp; i += MC_THREADS) {
            const int r = i / vp, c = (i - r * vp) * 4;
            mc_cp_async16(st_v + r * C + c, a.y.p + (r0 + r) * a.y.ld + vc + c);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // the gates of rows 2 lane and 2 lane + 1 (warp 0), a chunk ahead
    float li[2], lf[2];
    auto fetch_gates = [&](int chunk) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int r = chunk * R + 2 * lane + h;
            li[h] = -INFINITY;
            lf[h] = 0.f;
            if (r < n) {
                li[h] = log_input_gate(a, sl.first + r, head);
                lf[h] = log_forget_gate(a, sl.first + r, head);
            }
        }
    };
    if (chunks > 0) {
        if (staged) request(0);
        if (warp == 0) fetch_gates(0);
    }
    const float q_scale = rsqrtf((float)cm.dim);
    const int raw_width = cm.vdim;

    for (int ch = 0; ch < chunks; ++ch) {
        const int64_t r0 = sl.first + (int64_t)ch * R;
        const int m = min(R, n - ch * R);
        if (warp == 0) {
            // sums and running maxima of the chunk's rows, two per lane, in f64: differences of far sums stay exact
            double f1 = (double)lf[0] + lf[1];
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
            const double e_last = __shfl_sync(0xffffffffu, e[1], 31);  // rows past the end change neither sums nor maxima
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int r = 2 * lane + h;
                c_hi[r] = (float)c[h];
                c_lo[r] = c[h] == -INFINITY ? 0.f : (float)(c[h] - (double)c_hi[r]);
                e_hi[r] = (float)e[h];
                e_lo[r] = (float)(e[h] - (double)e_hi[r]);
                s_g[r] = expf((float)(run_max - e[h]));
                s_w[r] = expf((float)(c[h] - e_last));
                s_floor[r] = expf(-mt[h]);
            }
            if (lane == 0) *s_keep = expf((float)(run_max - e_last));
            run_max = __shfl_sync(0xffffffffu, mt[1], 31);
        }
        // q, k, v as bfloat16, rows past the end as zeros
        if (staged) asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the staged rows, the gates; everyone is through with the chunk before
        if (staged) {
            for (int i = threadIdx.x; i < R * (KD / 4); i += MC_THREADS) {
                const int r = i / (KD / 4), c = (i - r * (KD / 4)) * 4;
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
                if (r < m && c < cm.dim) {
                    x = *reinterpret_cast<const float4*>(st_q + r * KD + c);
                    y = *reinterpret_cast<const float4*>(st_k + r * KD + c);
                }
                const __nv_bfloat162 x0 = __floats2bfloat162_rn(x.x, x.y), x1 = __floats2bfloat162_rn(x.z, x.w);
                const __nv_bfloat162 y0 = __floats2bfloat162_rn(y.x, y.y), y1 = __floats2bfloat162_rn(y.z, y.w);
                *reinterpret_cast<uint2*>(Q + r * KP + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&x0), *reinterpret_cast<const uint32_t*>(&x1));
                *reinterpret_cast<uint2*>(K + r * KP + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&y0), *reinterpret_cast<const uint32_t*>(&y1));
            }
        } else {
            for (int i = threadIdx.x; i < R * KD; i += MC_THREADS) {
                const int r = i / KD, c = i - r * KD;
                const bool live = r < m && c < cm.dim;
                Q[r * KP + c] = __float2bfloat16_rn(live ? a.y.at(r0 + r, qc + c) : 0.f);
                K[r * KP + c] = __float2bfloat16_rn(live ? a.y.at(r0 + r, kc + c) : 0.f);
            }
        }
        for (int i = threadIdx.x; i < R * (C / 2); i += MC_THREADS) {
            const int r = i / (C / 2), c = (i - r * (C / 2)) * 2;
            float x = 0.f, y = 0.f;
            if (r < m) {
                if (c < cols) x = staged ? st_v[r * C + c] : a.y.at(r0 + r, vc + c);
                if (c + 1 < cols) y = staged ? st_v[r * C + c + 1] : a.y.at(r0 + r, vc + c + 1);
            }
            const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
            *reinterpret_cast<__nv_bfloat162*>(V + r * CP + c) = v;
            uint32_t hi, lo;
            mc_split(s_w[r] * __low2float(v), s_w[r] * __high2float(v), hi, lo);
            *reinterpret_cast<uint32_t*>(Wh + r * CP + c) = hi;
            *reinterpret_cast<uint32_t*>(Wl + r * CP + c) = lo;
        }
        __syncthreads();  // the staging rows are free, the operands are there
        if (ch + 1 < chunks) {
            if (staged) request(ch + 1);
            if (warp == 0) fetch_gates(ch + 1);
        }

        // D (Q K^T): 16 rows x 32 keys per warp, keys behind the rows are zeros
        {
            float sc[4][4] = {};
            const int k0 = half * 32;
            if (k0 <= row0 + 15) {
#pragma unroll
                for (int kk = 0; kk < KD / 16; ++kk) {
                    uint32_t af[4];
                    mc_ldmatrix(af, Q + (row0 + (lane & 15)) * KP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
                    for (int j = 0; j < 4; j += 2) {
                        uint32_t bf[4];
                        mc_ldmatrix(bf, K + (k0 + j * 8 + (lane & 7) + (lane >> 4) * 8) * KP + kk * 16 + ((lane >> 3) & 1) * 8);
                        mc_mma(sc[j], af, bf[0], bf[1]);
                        mc_mma(sc[j + 1], af, bf[2], bf[3]);
                    }
                }
            }
            float sum[2] = {0.f, 0.f};
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int t = row0 + gid + 8 * h, s = k0 + j * 8 + 2 * tq;
                    float p[2];
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        const float d = s + x <= t ? expf((c_hi[s + x] - e_hi[t]) + (c_lo[s + x] - e_lo[t])) : 0.f;
                        p[x] = sc[j][2 * h + x] * q_scale * d;
                        sum[h] += p[x];
                    }
                    uint32_t hi, lo;
                    mc_split(p[0], p[1], hi, lo);
                    *reinterpret_cast<uint32_t*>(Ph + t * PP + s) = hi;
                    *reinterpret_cast<uint32_t*>(Pl + t * PP + s) = lo;
                }
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 1);
                sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 2);
                if (tq == 0) s_sum[half * R + row0 + gid + 8 * h] = sum[h];
            }
            // n . q of the normaliser the chunk starts from: four threads per row
            const int t = threadIdx.x >> 2, part = threadIdx.x & 3;
            float nq = 0.f;
#pragma unroll 8
            for (int c = part * 2; c < KD; c += 8) {
                const __nv_bfloat162 q2 = *reinterpret_cast<const __nv_bfloat162*>(Q + t * KP + c);
                nq = fmaf(__low2float(q2), s_n[c], fmaf(__high2float(q2), s_n[c + 1], nq));
            }
            nq += __shfl_xor_sync(0xffffffffu, nq, 1);
            nq += __shfl_xor_sync(0xffffffffu, nq, 2);
            if (part == 0) s_nq[t] = nq;
        }
        __syncthreads();

        // outputs: 16 rows x C / 2 columns per warp
        {
            float o[NT][4] = {};
            const int n0 = half * (C / 2);
#pragma unroll
            for (int kk = 0; kk < KD / 16; ++kk) {
                uint32_t af[4];
                mc_ldmatrix(af, Q + (row0 + (lane & 15)) * KP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int j = 0; j < NT; j += 2) {
                    const int at = (n0 + j * 8 + (lane & 7) + (lane >> 4) * 8) * KP + kk * 16 + ((lane >> 3) & 1) * 8;
                    uint32_t bf[4];
                    mc_ldmatrix(bf, Sh + at);
                    mc_mma(o[j], af, bf[0], bf[1]);
                    mc_mma(o[j + 1], af, bf[2], bf[3]);
                    mc_ldmatrix(bf, Sl + at);
                    mc_mma(o[j], af, bf[0], bf[1]);
                    mc_mma(o[j + 1], af, bf[2], bf[3]);
                }
            }
            float g[2], den[2];
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int t = row0 + gid + 8 * h;
                g[h] = s_g[t] * q_scale;
                den[h] = fmaxf(fabsf(s_sum[t] + s_sum[R + t] + g[h] * s_nq[t]), s_floor[t]) + 1e-6f;
            }
#pragma unroll
            for (int j = 0; j < NT; ++j)
#pragma unroll
                for (int x = 0; x < 4; ++x) o[j][x] *= g[x >> 1];
            for (int kk = 0; kk <= (row0 >> 4); ++kk) {
                uint32_t ph[4], pl[4];
                const int at = (row0 + (lane & 15)) * PP + kk * 16 + (lane >> 4) * 8;
                mc_ldmatrix(ph, Ph + at);
                mc_ldmatrix(pl, Pl + at);
#pragma unroll
                for (int j = 0; j < NT; j += 2) {
                    uint32_t bf[4];
                    mc_ldmatrix_t(bf, V + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * CP + n0 + j * 8 + (lane >> 4) * 8);
                    mc_mma(o[j], ph, bf[0], bf[1]);
                    mc_mma(o[j + 1], ph, bf[2], bf[3]);
                    mc_mma(o[j], pl, bf[0], bf[1]);
                    mc_mma(o[j + 1], pl, bf[2], bf[3]);
                }
            }
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int t = row0 + gid + 8 * h;
                if (t >= m) continue;
                float* out = cm.out + ((r0 + t) * cm.heads + head) * raw_width + col0;
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    const int c = n0 + j * 8 + 2 * tq;
                    if (c < cols) out[c] = o[j][2 * h] / den[h];
                    if (c + 1 < cols) out[c + 1] = o[j][2 * h + 1] / den[h];
                }
            }
        }
        // the state behind the chunk: 16 columns x KEYS keys per warp
        const float keep = *s_keep;
#pragma unroll
        for (int j = 0; j < NK; ++j)
#pragma unroll
            for (int x = 0; x < 4; ++x) S[j][x] *= keep;
#pragma unroll
        for (int kk = 0; kk < R / 16; ++kk) {
            uint32_t wh[4], wl[4];
            const int at = (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * CP + sc0 + ((lane >> 3) & 1) * 8;
            mc_ldmatrix_t(wh, Wh + at);
            mc_ldmatrix_t(wl, Wl + at);
#pragma unroll
            for (int j = 0; j < NK; j += 2) {
                uint32_t bf[4];
                mc_ldmatrix_t(bf, K + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * KP + sk0 + j * 8 + (lane >> 4) * 8);
                mc_mma(S[j], wh, bf[0], bf[1]);
                mc_mma(S[j + 1], wh, bf[2], bf[3]);
                mc_mma(S[j], wl, bf[0], bf[1]);
                mc_mma(S[j + 1], wl, bf[2], bf[3]);
            }
        }
        for (int i = threadIdx.x; i < KD; i += MC_THREADS) {
            float x = s_n[i] * keep;
#pragma unroll 8
            for (int t = 0; t < R; ++t) x = fmaf(s_w[t], __bfloat162float(K[t * KP + i]), x);
            s_n[i] = x;  // read again behind the next barrier only
        }
        __syncthreads();  // the old state was read by everyone
        if (ch + 1 < chunks) publish_state();
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
        for (int i = threadIdx.x; i < KD; i += MC_THREADS) dst[(int64_t)cm.vdim * KD + i] = s_n[i];
        if (threadIdx.x == 0) a.running_max[(int64_t)sl.out * cm.heads + head] = run_max;
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
    const dim3 grid((unsigned)((c.vdim + C - 1) / C), (unsigned)c.heads, (unsigned)c.lanes.lanes);
    launch_pdl(kernel, grid, dim3(MC_THREADS), Chunk<KD, C>::BYTES, s, a, aligned_heads(a) && a.y.n == 1 ? 1 : 0);
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
