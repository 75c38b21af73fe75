// See linear_state.h.
//
// A group of KS threads holds two value columns of one (lane, head), the columns' keys shared out over the group's threads in
// runs of four; the state stays in registers while the lane's rows go by.  Rows arrive in shared memory in chunks, fetched with
// cp.async while the chunk before is being worked on, and a thread loads the next row's vectors while it works on the current
// one.  The sums over the keys of four rows are folded together (each exchange halves what is left), so a row costs under two
// shuffles per column pair - except the delta rule's S^T k, which the row itself depends on.  Wide prompts cut a head's columns
// over CTAs of four warps with sixteen threads per column pair (the delta rule's chain of dependent steps sets the pace there)
// and leave the head norm to a second kernel; ticks of short lanes give a whole head to one CTA, which then finishes the output
// row itself: there the state's way through the SM is what counts.
#include "linear_state.h"
#include "recurrent_core.cuh"
#include <algorithm>

namespace mk {

namespace {

constexpr int LS_WIDE_WARPS = 4;  // warps of a CTA that owns part of a head
constexpr int LS_MAX_FINISH_V = 128;

enum LsRule : int { LS_WKV, LS_DELTA, LS_MLSTM, LS_CHANNEL };
template <LsRule RULE>
struct LsArgs;
template <>
struct LsArgs<LS_WKV> { using type = WkvScanArgs; };
template <>
struct LsArgs<LS_DELTA> { using type = DeltaScanArgs; };
template <>
struct LsArgs<LS_MLSTM> { using type = MlstmScanArgs; };
template <>
struct LsArgs<LS_CHANNEL> { using type = ChannelDeltaArgs; };

__device__ __forceinline__ void ls_cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ls_cp_async4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ls_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void ls_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// `n` rows of `width` floats, row i from src(i), into dst rows `pitch` floats apart; `vec`: everything is 16-byte aligned.
template <typename Src>
__device__ __forceinline__ void fetch_rows(float* dst, int pitch, int n, int width, bool vec, Src src) {
    if (vec) {
        const int per = width >> 2;
        for (int i = threadIdx.x; i < n * per; i += blockDim.x) {
            const int r = i / per, c = (i - r * per) * 4;
            ls_cp_async16(dst + r * pitch + c, src(r) + c);
        }
    } else {
        for (int i = threadIdx.x; i < n * width; i += blockDim.x) {
            const int r = i / width, c = i - r * width;
            ls_cp_async4(dst + r * pitch + c, src(r) + c);
        }
    }
}
// The same rows of a matmul output that is still in shares.
__device__ __forceinline__ void sum_rows(float* dst, int pitch, int n, int width, const Shares& y, int64_t row0, int col) {
    for (int i = threadIdx.x; i < n * width; i += blockDim.x) {
        const int r = i / width, c = i - r * width;
        dst[r * pitch + c] = y.at(row0 + r, col + c);
    }
}

// Eight values per thread, folded over the KS threads of a group: thread t ends with the sum of value t % 8.
template <int KS>
__device__ __forceinline__ float fold8(const float (&v)[8], int t) {
    float a[4], b[2];
    const bool h4 = (t & 4) != 0, h2 = (t & 2) != 0, h1 = (t & 1) != 0;
#pragma unroll
    for (int i = 0; i < 4; ++i) a[i] = (h4 ? v[i + 4] : v[i]) + __shfl_xor_sync(0xffffffffu, h4 ? v[i] : v[i + 4], 4);
#pragma unroll
    for (int i = 0; i < 2; ++i) b[i] = (h2 ? a[i + 2] : a[i]) + __shfl_xor_sync(0xffffffffu, h2 ? a[i] : a[i + 2], 2);
    float r = (h1 ? b[1] : b[0]) + __shfl_xor_sync(0xffffffffu, h1 ? b[0] : b[1], 1);
#pragma unroll
    for (int x = 8; x < KS; x <<= 1) r += __shfl_xor_sync(0xffffffffu, r, x);
    return r;
}

// One head's row o[0 .. vdim) of packed row `row`, by one warp; gate[v] and norm weights nw[v] of the head, den: its denominator.
template <typename Gate>
__device__ __forceinline__ void finish_head_row(const LinearStateArgs& a, const float* o, float den, Gate gate, const float* nw, int64_t row, int head, int lane) {
    float ss = 0.f;
    for (int v = lane; v < a.vdim; v += 32) ss += (o[v] / den) * (o[v] / den);
    ss = warp_sum(ss);
    const float root = sqrtf(ss / (float)a.vdim + a.eps);
    for (int v = lane; v < a.vdim; v += 32) {
        const float g = gate(v);
        a.image.put(row, head * a.vdim + v, o[v] / den / root * nw[v] * (a.gate_sigmoid ? sigmoid_f(g) : silu_f(g)) * a.out_scale);
    }
    if (head == a.heads - 1)
        for (int c = a.heads * a.vdim + lane; c < a.image.end(); c += 32) a.image.put(row, c, 0.f);
}

template <int KD, LsRule RULE, bool FINISH>
struct Ls {
    static constexpr bool WKV = RULE == LS_WKV, CHANNEL = RULE == LS_CHANNEL;
    static constexpr bool ROW_DECAY = WKV || CHANNEL;        // a decay per key, as a row of its own
    static constexpr int EXTRA = RULE == LS_MLSTM ? 1 : 0;   // columns of the state beside the values
    static constexpr int KS = !FINISH && KD >= 64 ? 16 : 8;  // threads of a column pair
    static constexpr int KE = KD / KS;                       // keys of a thread
    static constexpr int COLS = 32 / KS * 2;                 // value columns of a warp
    static constexpr int TT = FINISH ? 4 : 16;               // rows of a chunk
    static constexpr int KROWS = CHANNEL ? 4 : (WKV ? 3 : 2);  // r, k, decay, removal  /  r, k, decay  /  q, k
    static constexpr int MAX_THREADS = FINISH ? LS_MAX_FINISH_V / COLS * 32 : LS_WIDE_WARPS * 32;
    static constexpr int MIN_CTAS = FINISH && !CHANNEL ? (KD >= 128 ? 2 : 3) : 1;
    // stage: KROWS key-wide rows, the value row, the gate row (FINISH), decay, write and floor of the denominator (not ROW_DECAY)
    static __host__ __device__ constexpr int row_floats(int cols) { return KROWS * KD + cols * (FINISH ? 2 : 1) + (ROW_DECAY ? 0 : 4); }
    static __host__ __device__ constexpr int stage_floats(int cols) { return TT * row_floats(cols); }
    // two stages; FINISH: the output rows and the head's norm weights
    static __host__ __device__ constexpr size_t bytes(int cols) { return (2 * (size_t)stage_floats(cols) + (FINISH ? (size_t)(TT + 1) * cols : 0)) * 4; }
};

template <int KD, LsRule RULE, bool FINISH>
__global__ void __launch_bounds__(Ls<KD, RULE, FINISH>::MAX_THREADS, Ls<KD, RULE, FINISH>::MIN_CTAS)
linear_state_kernel(const __grid_constant__ typename LsArgs<RULE>::type ra) {
    using L = Ls<KD, RULE, FINISH>;
    constexpr bool WKV = L::WKV, CHANNEL = L::CHANNEL, ROW_DECAY = L::ROW_DECAY;
    constexpr int TT = L::TT, KS = L::KS, KE = L::KE, NJ = KE / 4;
    extern __shared__ __align__(16) float ls_smem[];
    const LinearStateArgs& a = ra.common;
    const int state_cols = a.vdim + L::EXTRA;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ks = lane & (KS - 1);
    const int cols = (int)(blockDim.x >> 5) * L::COLS;                 // columns of this CTA
    const int col0 = blockIdx.x * cols;
    const int head = blockIdx.y;
    const int c_loc = warp * L::COLS + lane / KS * 2;                  // first of the thread's two columns, within the CTA
    const int my_cols = max(0, min(cols, a.vdim - col0));              // of them values
    float* s_o = ls_smem + 2 * L::stage_floats(cols);                  // FINISH: [TT][cols]
    float* s_nw = s_o + TT * cols;                                     // FINISH: [cols]

    // The lane record was staged by the host, weights never change and the committed state was written by an earlier tick: none
    // of them depends on the predecessor kernel, so all are on their way before the wait.
    pdl_trigger();
    const StateLane sl = a.lanes.at(blockIdx.z);
    float S[2][KE];
    const int64_t head_state = (int64_t)state_cols * KD;
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        const int v = col0 + c_loc + c;
        const bool live = sl.in >= 0 && v < state_cols;
        const float4* src = reinterpret_cast<const float4*>(a.state + ((int64_t)sl.in * a.heads + head) * head_state + (int64_t)v * KD);
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const float4 x = live ? __ldcs(src + j * KS + ks) : make_float4(0.f, 0.f, 0.f, 0.f);
            S[c][4 * j] = x.x; S[c][4 * j + 1] = x.y; S[c][4 * j + 2] = x.z; S[c][4 * j + 3] = x.w;
        }
    }
    float U[WKV ? KE : 1];
    if constexpr (WKV) {
#pragma unroll
        for (int e = 0; e < KE; ++e) {
            const int i = (e >> 2) * 4 * KS + ks * 4 + (e & 3);
            U[e] = i < a.dim ? ra.bonus[head * a.dim + i] : 0.f;
        }
    }
    // mLSTM: the first warp turns the gates of a chunk's rows into decay, write and floor, a row per lane
    float run_max = 0.f;
    if constexpr (RULE == LS_MLSTM) {
        if (warp == 0 && sl.in >= 0) run_max = ra.running_max[(int64_t)sl.in * a.heads + head];
    }
    if (FINISH)
        for (int v = threadIdx.x; v < a.vdim; v += blockDim.x) s_nw[v] = a.norm_w[(a.norm_per_head ? head * a.vdim : 0) + v];
    // key columns past the true dimension and value columns past the last stay zero in both stages
    if (a.dim < KD || my_cols < cols) {
        for (int i = threadIdx.x; i < 2 * L::stage_floats(cols); i += blockDim.x) ls_smem[i] = 0.f;
        __syncthreads();
    }
    if (RULE == LS_MLSTM && a.vdim >= col0 && a.vdim < col0 + cols)  // the normaliser's value
        for (int i = threadIdx.x; i < 2 * TT; i += blockDim.x)
            ls_smem[i / TT * L::stage_floats(cols) + TT * L::KROWS * KD + i % TT * cols + a.vdim - col0] = 1.f;
    pdl_wait();

    const int first = sl.first, n = sl.n;
    const bool vec = (a.dim & 3) == 0 && (a.vdim & 3) == 0;
    const int raw_width = RULE == LS_MLSTM ? linear_state_raw_width(a.vdim) : a.vdim;
    const float q_scale = RULE == LS_MLSTM ? rsqrtf((float)a.dim) : 1.f;
    auto stage = [&](int which) { return ls_smem + which * L::stage_floats(cols); };
    auto fetch = [&](int chunk) {
        float* s = stage(chunk & 1);
        const int64_t r0 = first + chunk * TT;
        const int m = min(TT, n - chunk * TT);
        float* s_v = s + TT * L::KROWS * KD;
        float* s_g = s_v + TT * cols;
        float* s_c = s_v + TT * cols * (FINISH ? 2 : 1);
        // the first key-wide row, the second and the values, from a matmul's output
        auto fetch_heads = [&](const Shares& y, int x_col, int k_col, int v_col) {
            if (y.n == 1) {
                const bool yv = vec && (y.ld & 3) == 0;
                fetch_rows(s, KD, m, a.dim, yv, [&](int r) { return y.p + (r0 + r) * y.ld + x_col; });
                fetch_rows(s + TT * KD, KD, m, a.dim, yv, [&](int r) { return y.p + (r0 + r) * y.ld + k_col; });
                fetch_rows(s_v, cols, m, my_cols, yv && (my_cols & 3) == 0, [&](int r) { return y.p + (r0 + r) * y.ld + v_col; });
            } else {
                sum_rows(s, KD, m, a.dim, y, r0, x_col);
                sum_rows(s + TT * KD, KD, m, a.dim, y, r0, k_col);
                sum_rows(s_v, cols, m, my_cols, y, r0, v_col);
            }
        };
        if constexpr (RULE == LS_WKV) {
            const int h0 = head * a.dim;
            fetch_heads(ra.rkv, ra.r_col + h0, ra.k_col + h0, ra.v_col + h0 + col0);
            fetch_rows(s + 2 * TT * KD, KD, m, a.dim, vec, [&](int r) { return ra.decay + (r0 + r) * a.heads * a.dim + h0; });
        } else if constexpr (CHANNEL) {
            const int h0 = head * a.dim;
            fetch_heads(ra.y, ra.r_col + h0, ra.k_col + h0, ra.v_col + head * a.vdim + col0);
            fetch_rows(s + 2 * TT * KD, KD, m, a.dim, vec, [&](int r) { return ra.decay + (r0 + r) * a.heads * a.dim + h0; });
            fetch_rows(s + 3 * TT * KD, KD, m, a.dim, vec, [&](int r) { return ra.removal + (r0 + r) * a.heads * a.dim + h0; });
        } else if constexpr (RULE == LS_MLSTM) {
            const int h0 = head * a.dim;
            fetch_heads(ra.y, ra.q_col + h0, ra.k_col + h0, ra.v_col + head * a.vdim + col0);
            if (warp == 0) {
                float f = 0.f, i = -INFINITY;
                if (lane < m) {
                    i = ra.cap * tanhf((ra.y.at(r0 + lane, ra.i_col + head) + ra.i_bias[head]) / ra.cap);
                    f = -recurrent::softplus_stable(-ra.cap * tanhf((ra.y.at(r0 + lane, ra.f_col + head) + ra.f_bias[head]) / ra.cap));
                }
                // row t's maximum is max(sum of f up to t + the chunk's first maximum, running maximum of i with f added since)
                float sum = f, top = i;
#pragma unroll
                for (int o = 1; o < TT; o <<= 1) {
                    const float ps = __shfl_up_sync(0xffffffffu, sum, o), pt = __shfl_up_sync(0xffffffffu, top, o);
                    if (lane >= o) {
                        top = fmaxf(pt + sum, top);
                        sum += ps;
                    }
                }
                const float mt = fmaxf(run_max + sum, top);
                float before = __shfl_up_sync(0xffffffffu, mt, 1);
                if (lane == 0) before = run_max;
                if (lane < m) {
                    s_c[4 * lane] = expf(f + before - mt);
                    s_c[4 * lane + 1] = expf(i - mt);
                    s_c[4 * lane + 2] = expf(-mt);
                }
                run_max = __shfl_sync(0xffffffffu, mt, m - 1);
            }
        } else {
            const int kv_head = head / (a.heads / ra.kv_heads);
            const int64_t kw = (int64_t)ra.kv_heads * a.dim, vw = (int64_t)a.heads * a.vdim;
            fetch_rows(s, KD, m, a.dim, vec, [&](int r) { return ra.q + (r0 + r) * kw + kv_head * a.dim; });
            fetch_rows(s + TT * KD, KD, m, a.dim, vec, [&](int r) { return ra.k + (r0 + r) * kw + kv_head * a.dim; });
            fetch_rows(s_v, cols, m, my_cols, vec && (my_cols & 3) == 0, [&](int r) { return ra.v + (r0 + r) * vw + head * a.vdim + col0; });
            for (int r = threadIdx.x; r < m; r += blockDim.x) {
                ls_cp_async4(s_c + 4 * r, ra.decay + (r0 + r) * a.heads + head);
                ls_cp_async4(s_c + 4 * r + 1, ra.beta + (r0 + r) * a.heads + head);
            }
        }
        if (FINISH) sum_rows(s_g, cols, m, a.vdim, a.gate, r0, a.gate_col + head * a.vdim);
        ls_commit();
    };

    const int chunks = (n + TT - 1) / TT;
    if (chunks > 0) fetch(0);
    for (int ch = 0; ch < chunks; ++ch) {
        if (ch + 1 < chunks) {
            fetch(ch + 1);
            ls_wait<1>();
        } else {
            ls_wait<0>();
        }
        float* s = stage(ch & 1);
        float* s_v = s + TT * L::KROWS * KD;
        float* s_c = s_v + TT * cols * (FINISH ? 2 : 1);
        const int m = min(TT, n - ch * TT);
        if (!FINISH && (m & 3) != 0) {
            // rows are taken four at a time: those past the last one change nothing (k = 0, no decay)
            __syncthreads();
            for (int t = m; t < ((m + 3) & ~3); ++t) {
                for (int i = threadIdx.x; i < KD; i += blockDim.x) {
                    s[t * KD + i] = 0.f;
                    s[TT * KD + t * KD + i] = 0.f;
                    if (ROW_DECAY) s[2 * TT * KD + t * KD + i] = 1.f;
                    if (CHANNEL) s[3 * TT * KD + t * KD + i] = 0.f;
                }
                for (int i = threadIdx.x; i < cols; i += blockDim.x) s_v[t * cols + i] = 0.f;
                if (!ROW_DECAY && threadIdx.x == 0) {
                    s_c[4 * t] = 1.f;
                    s_c[4 * t + 1] = 0.f;
                }
            }
        }
        __syncthreads();
        // one row's vectors: r | q in x, k in y, decay in w (WKV, CHANNEL), removal in b (CHANNEL)
        struct Row {
            float x[KE], y[KE], w[ROW_DECAY ? KE : 1], b[CHANNEL ? KE : 1];
            float2 v, gb;
        };
        auto load_row = [&](int t, Row& r) {
            const float4* x4 = reinterpret_cast<const float4*>(s + t * KD) + ks;
            const float4* y4 = reinterpret_cast<const float4*>(s + TT * KD + t * KD) + ks;
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const float4 y = y4[j * KS], x = x4[j * KS];
                r.y[4 * j] = y.x; r.y[4 * j + 1] = y.y; r.y[4 * j + 2] = y.z; r.y[4 * j + 3] = y.w;
                r.x[4 * j] = x.x; r.x[4 * j + 1] = x.y; r.x[4 * j + 2] = x.z; r.x[4 * j + 3] = x.w;
            }
            if constexpr (ROW_DECAY) {
                const float4* w4 = reinterpret_cast<const float4*>(s + 2 * TT * KD + t * KD) + ks;
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const float4 w = w4[j * KS];
                    r.w[4 * j] = w.x; r.w[4 * j + 1] = w.y; r.w[4 * j + 2] = w.z; r.w[4 * j + 3] = w.w;
                }
            } else {
                r.gb = *reinterpret_cast<const float2*>(s_c + 4 * t);
            }
            if constexpr (CHANNEL) {
                const float4* b4 = reinterpret_cast<const float4*>(s + 3 * TT * KD + t * KD) + ks;
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const float4 b = b4[j * KS];
                    r.b[4 * j] = b.x; r.b[4 * j + 1] = b.y; r.b[4 * j + 2] = b.z; r.b[4 * j + 3] = b.w;
                }
            }
            r.v = *reinterpret_cast<const float2*>(s_v + t * cols + c_loc);
        };
        auto step = [&](const Row& r, float& out0, float& out1) {
            float o0 = 0.f, o1 = 0.f;
            if constexpr (RULE == LS_MLSTM) {
                const float u0 = r.gb.y * r.v.x, u1 = r.gb.y * r.v.y;
#pragma unroll
                for (int e = 0; e < KE; ++e) {
                    S[0][e] = fmaf(r.y[e], u0, r.gb.x * S[0][e]);
                    S[1][e] = fmaf(r.y[e], u1, r.gb.x * S[1][e]);
                    o0 = fmaf(S[0][e], r.x[e], o0);
                    o1 = fmaf(S[1][e], r.x[e], o1);
                }
            } else if constexpr (WKV) {
#pragma unroll
                for (int e = 0; e < KE; ++e) {
                    const float uk = U[e] * r.y[e];
                    o0 = fmaf(r.x[e], fmaf(uk, r.v.x, S[0][e]), o0);
                    o1 = fmaf(r.x[e], fmaf(uk, r.v.y, S[1][e]), o1);
                    S[0][e] = fmaf(r.w[e], S[0][e], r.y[e] * r.v.x);
                    S[1][e] = fmaf(r.w[e], S[1][e], r.y[e] * r.v.y);
                }
            } else {
                float d0[2] = {0.f, 0.f}, d1[2] = {0.f, 0.f};
#pragma unroll
                for (int e = 0; e < KE; ++e) {
                    d0[e & 1] = fmaf(S[0][e], r.y[e], d0[e & 1]);
                    d1[e & 1] = fmaf(S[1][e], r.y[e], d1[e & 1]);
                }
                float m0 = d0[0] + d0[1], m1 = d1[0] + d1[1];
#pragma unroll
                for (int x = 1; x < KS; x <<= 1) {
                    m0 += __shfl_xor_sync(0xffffffffu, m0, x);
                    m1 += __shfl_xor_sync(0xffffffffu, m1, x);
                }
                if constexpr (CHANNEL) {
#pragma unroll
                    for (int e = 0; e < KE; ++e) {
                        S[0][e] = fmaf(-r.b[e], m0, fmaf(r.w[e], S[0][e], r.y[e] * r.v.x));
                        S[1][e] = fmaf(-r.b[e], m1, fmaf(r.w[e], S[1][e], r.y[e] * r.v.y));
                        o0 = fmaf(S[0][e], r.x[e], o0);
                        o1 = fmaf(S[1][e], r.x[e], o1);
                    }
                    out0 = o0;
                    out1 = o1;
                    return;
                }
                const float u0 = r.gb.y * (r.v.x - r.gb.x * m0), u1 = r.gb.y * (r.v.y - r.gb.x * m1);
#pragma unroll
                for (int e = 0; e < KE; ++e) {
                    S[0][e] = fmaf(r.y[e], u0, r.gb.x * S[0][e]);
                    S[1][e] = fmaf(r.y[e], u1, r.gb.x * S[1][e]);
                    o0 = fmaf(S[0][e], r.x[e], o0);
                    o1 = fmaf(S[1][e], r.x[e], o1);
                }
            }
            out0 = o0;
            out1 = o1;
        };
        if constexpr (FINISH) {
            float part[8];
            Row r;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                part[2 * i] = part[2 * i + 1] = 0.f;
                if (i < m) {  // uniform over the CTA
                    load_row(i, r);
                    step(r, part[2 * i], part[2 * i + 1]);
                }
            }
            const float o = fold8<KS>(part, ks);
            const int t = ks >> 1, c = c_loc + (ks & 1);
            if (t < m && c < a.vdim) s_o[t * cols + c] = o;
            __syncthreads();
            const float* s_g = s_v + TT * cols;
            for (int t = warp; t < m; t += (int)(blockDim.x >> 5))
                finish_head_row(a, s_o + t * cols, 1.f, [&](int v) { return s_g[t * cols + v]; }, s_nw, first + ch * TT + t, head, lane);
            __syncthreads();  // the stage is free for the chunk after next
        } else {
            Row rows[2];
            load_row(0, rows[0]);
#pragma unroll 1
            for (int t0 = 0; t0 < m; t0 += 4) {
                float part[8];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    load_row(min(t0 + i + 1, TT - 1), rows[(i + 1) & 1]);
                    step(rows[i & 1], part[2 * i], part[2 * i + 1]);
                }
                float o = fold8<KS>(part, ks);
                const int t = t0 + ((ks & 7) >> 1), c = c_loc + (ks & 1);
                if (RULE == LS_MLSTM) {
                    o *= q_scale;
                    if (col0 + c == a.vdim && t < m) o = fmaxf(fabsf(o), s_c[4 * t + 2]) + 1e-6f;
                }
                if (ks < 8 && t < m && col0 + c < state_cols)
                    a.out[((int64_t)(first + ch * TT + t) * a.heads + head) * raw_width + col0 + c] = o;
            }
            __syncthreads();  // the stage is free for the chunk after next
        }
    }

#pragma unroll
    for (int c = 0; c < 2; ++c) {
        const int v = col0 + c_loc + c;
        if (v >= state_cols) continue;
        float4* dst = reinterpret_cast<float4*>(a.state + ((int64_t)sl.out * a.heads + head) * head_state + (int64_t)v * KD);
#pragma unroll
        for (int j = 0; j < NJ; ++j) __stcs(dst + j * KS + ks, make_float4(S[c][4 * j], S[c][4 * j + 1], S[c][4 * j + 2], S[c][4 * j + 3]));
    }
    if constexpr (RULE == LS_MLSTM) {
        if (blockIdx.x == 0 && threadIdx.x == 0) ra.running_max[(int64_t)sl.out * a.heads + head] = run_max;
    }
}

__global__ void __launch_bounds__(128) head_norm_gate_kernel(LinearStateArgs a, int rows) {
    pdl_trigger();
    pdl_wait();
    const int64_t i = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (i >= (int64_t)rows * a.heads) return;
    const int64_t row = i / a.heads;
    const int head = (int)(i % a.heads);
    const int width = a.normalised ? linear_state_raw_width(a.vdim) : a.vdim;
    const float* o = a.out + (row * a.heads + head) * width;
    finish_head_row(a, o, a.normalised ? o[a.vdim] : 1.f, [&](int v) { return a.gate.at(row, a.gate_col + head * a.vdim + v); },
                    a.norm_w + (a.norm_per_head ? head * a.vdim : 0), row, head, threadIdx.x & 31);
}

// The same with four values per thread and G threads per head row (vdim a multiple of 4, at most 4 G): narrow heads share a warp.
template <int G>
__global__ void __launch_bounds__(128) head_norm_gate_vec_kernel(LinearStateArgs a, int rows) {
    pdl_trigger();
    pdl_wait();
    const int64_t i = (int64_t)blockIdx.x * (128 / G) + threadIdx.x / G;
    const bool live = i < (int64_t)rows * a.heads;
    const int64_t row = live ? i / a.heads : 0;
    const int head = live ? (int)(i % a.heads) : 0, v = (int)(threadIdx.x % G) * 4;
    const bool mine = live && v < a.vdim;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f), g = o, w = o;
    if (mine) {
        const float* src = a.out + (row * a.heads + head) * (a.normalised ? linear_state_raw_width(a.vdim) : a.vdim);
        o = *reinterpret_cast<const float4*>(src + v);
        if (a.normalised) {
            const float den = src[a.vdim];
            o = make_float4(o.x / den, o.y / den, o.z / den, o.w / den);
        }
        g = a.gate.at4(row, a.gate_col + head * a.vdim + v);
        w = *reinterpret_cast<const float4*>(a.norm_w + (a.norm_per_head ? head * a.vdim : 0) + v);
    }
    float ss = o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w;
#pragma unroll
    for (int x = 1; x < G; x <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    const float root = sqrtf(ss / (float)a.vdim + a.eps);
    if (mine) {
        w = make_float4(w.x * a.out_scale, w.y * a.out_scale, w.z * a.out_scale, w.w * a.out_scale);
        g = a.gate_sigmoid ? make_float4(sigmoid_f(g.x), sigmoid_f(g.y), sigmoid_f(g.z), sigmoid_f(g.w)) : make_float4(silu_f(g.x), silu_f(g.y), silu_f(g.z), silu_f(g.w));
        a.image.put4(row, head * a.vdim + v, make_float4(o.x / root * w.x * g.x, o.y / root * w.y * g.y, o.z / root * w.z * g.z, o.w / root * w.w * g.w));
    }
    if (live && head == a.heads - 1)
        for (int c = a.heads * a.vdim + (int)(threadIdx.x % G); c < a.image.end(); c += G) a.image.put(row, c, 0.f);
}

template <int KD, LsRule RULE, bool FINISH>
void launch_variant(const typename LsArgs<RULE>::type& ra, cudaStream_t s) {
    const LinearStateArgs& a = ra.common;
    using L = Ls<KD, RULE, FINISH>;
    const int state_cols = a.vdim + L::EXTRA;
    const int warps = FINISH ? (state_cols + L::COLS - 1) / L::COLS : LS_WIDE_WARPS;
    const int cols = warps * L::COLS;
    const size_t smem = L::bytes(cols);
    auto* kernel = linear_state_kernel<KD, RULE, FINISH>;
    ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), smem);
    const dim3 grid((unsigned)((state_cols + cols - 1) / cols), (unsigned)a.heads, (unsigned)a.lanes.lanes);
    launch_pdl(kernel, grid, dim3((unsigned)warps * 32), smem, s, ra);
    MK_LAUNCH_CHECK();
}

template <LsRule RULE>
void launch_scan(const typename LsArgs<RULE>::type& ra, cudaStream_t s) {
    const LinearStateArgs& a = ra.common;
    if (a.lanes.lanes <= 0) return;
    if (a.heads > 65535 || a.lanes.lanes > 65535) throw std::runtime_error("linear-attention scan: at most 65535 heads and lanes");
    const bool finish = a.image.h != nullptr || a.image.f != nullptr;
    if (finish && !linear_state_can_finish(a.dim, a.vdim)) throw std::runtime_error("linear-attention scan: the finishing form takes dimensions up to 128");
    const int pad = linear_state_key_pad(a.dim);
    if constexpr (RULE != LS_MLSTM) {
        if (finish) {
            if (pad == 32) launch_variant<32, RULE, true>(ra, s);
            else if (pad == 64) launch_variant<64, RULE, true>(ra, s);
            else launch_variant<128, RULE, true>(ra, s);
            return;
        }
    }
    switch (pad) {
        case 32: launch_variant<32, RULE, false>(ra, s); break;
        case 64: launch_variant<64, RULE, false>(ra, s); break;
        case 128: launch_variant<128, RULE, false>(ra, s); break;
        default: launch_variant<256, RULE, false>(ra, s); break;
    }
}

}  // namespace

int linear_state_key_pad(int dim) {
    for (int p : {32, 64, 128, 256})
        if (dim <= p) return p;
    throw std::runtime_error("a recurrent head dimension above 256 is not supported");
}

bool linear_state_can_finish(int dim, int vdim) { return dim <= 128 && vdim <= LS_MAX_FINISH_V; }

void launch_wkv_scan(const WkvScanArgs& a, cudaStream_t s) { launch_scan<LS_WKV>(a, s); }

int launch_mlstm_scan(const MlstmScanArgs& a, cudaStream_t s) {
    if (a.longest <= 1 && a.yh == nullptr) {
        launch_mlstm_step(a, s);
        return 1;
    }
    MlstmScanArgs raw = a;
    raw.common.image = RowImage{};
    LinearStateArgs finish = a.common;
    if (a.yh != nullptr) {
        launch_mlstm_chunks(raw, s);
    } else {
        launch_scan<LS_MLSTM>(raw, s);
        finish.normalised = 1;
    }
    launch_head_norm_gate(finish, a.rows, s);
    return 2;
}

void launch_delta_scan(const DeltaScanArgs& a, cudaStream_t s) {
    if (a.kv_heads <= 0 || a.common.heads % a.kv_heads != 0) throw std::runtime_error("delta-rule scan: heads must be a multiple of kv_heads");
    launch_scan<LS_DELTA>(a, s);
}

void launch_channel_delta_scan(const ChannelDeltaArgs& a, cudaStream_t s) {
    if (a.common.dim != a.common.vdim) throw std::runtime_error("delta-rule scan with channel gates: square heads only");
    launch_scan<LS_CHANNEL>(a, s);
}

void launch_head_norm_gate(const LinearStateArgs& a, int rows, cudaStream_t s) {
    if (rows <= 0) return;
    const int64_t items = (int64_t)rows * a.heads;
    const bool vec = a.vdim % 4 == 0 && a.vdim <= 128 && a.gate_col % 4 == 0 && a.gate.ld % 4 == 0 && a.gate.stride % 4 == 0 &&
                     (reinterpret_cast<uintptr_t>(a.gate.p) & 15) == 0;
    if (vec && a.vdim <= 64) launch_pdl(head_norm_gate_vec_kernel<16>, dim3((unsigned)((items + 7) / 8)), dim3(128), 0, s, a, rows);
    else if (vec) launch_pdl(head_norm_gate_vec_kernel<32>, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, s, a, rows);
    else launch_pdl(head_norm_gate_kernel, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, s, a, rows);
    MK_LAUNCH_CHECK();
}

}  // namespace mk
