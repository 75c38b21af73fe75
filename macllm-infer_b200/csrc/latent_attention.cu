// See latent_attention.h.
//
// Tensor-core kernel: one CTA per (query row, share of its keys, up to 32 heads).  The four warps each own a quarter of the
// latent's columns: a warp's cp.async ring holds its columns of the next tiles of 32 rows, its queries' columns stay in registers,
// its partial scores meet the other warps' in shared memory (the one barrier of a tile, double-buffered), every warp then forms
// the same softmax weights and adds up its columns of the output from the rows it already holds.  A row is thus read once for
// keys and values, and by one warp per column.  Scores, softmax and sums are f32; the weights enter the second product as the sum
// of two f16 numbers.  When few rows are in flight their keys are shared out over several CTAs; the one that finishes last adds
// the shares in order.
#include "latent_attention.h"
#include "device_util.h"
#include <algorithm>

namespace mk {

namespace {

constexpr int LA_WARPS = 4;
constexpr int LA_KT = 32;             // keys of a tile
constexpr int LA_STAGES = 2;
constexpr int LA_SP = LA_KT + 4;      // pitch of the partial scores
constexpr int LA_SMS = 148;
constexpr int LA_TARGET_CTAS = LA_SMS * 2;
constexpr int LA_MIN_SHARE = 256;
constexpr int LA_MAX_SHARES = 32;
constexpr int LA_SHARED_ROWS = 256;   // ticks with more query rows are not cut into shares

__device__ __forceinline__ uint32_t la_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void la_ldm4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(la_smem(p)));
}
__device__ __forceinline__ void la_ldm4_trans(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(la_smem(p)));
}
__device__ __forceinline__ void la_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t la_pack(float x, float y) {
    const __half2 h = __floats2half2_rn(x, y);
    return *reinterpret_cast<const uint32_t*>(&h);
}
// What f16 rounding left of two weights.
__device__ __forceinline__ uint32_t la_rest(float x, float y, uint32_t rounded) {
    const float2 r = __half22float2(*reinterpret_cast<const __half2*>(&rounded));
    return la_pack(x - r.x, y - r.y);
}

struct LatentEntry {
    int row, share, n_shares, pos, table_off, packed, first;
};
__device__ __forceinline__ LatentEntry load_entry(const int32_t* entries, int i) {
    const int4 a = reinterpret_cast<const int4*>(entries)[2 * i], b = reinterpret_cast<const int4*>(entries)[2 * i + 1];
    return LatentEntry{a.x, a.y, a.z, a.w, b.x, b.y, b.z};
}

template <int RANK, int MT>
struct La {
    static constexpr int CW = RANK / LA_WARPS;   // columns of a warp
    static constexpr int PITCH = CW + 8;         // halves: conflict-free ldmatrix
    static constexpr int KS = CW / 16;
    static constexpr int NT = CW / 8;
    static constexpr int STAGE = LA_KT * PITCH;  // halves of a warp's stage
    static constexpr int SCORES = LA_WARPS * MT * 16 * LA_SP;
    static constexpr size_t BYTES = (size_t)LA_WARPS * LA_STAGES * STAGE * 2 + (size_t)2 * SCORES * 4;
};

template <int RANK, int MT>
__global__ void __launch_bounds__(LA_WARPS * 32, 2) latent_tc_kernel(LatentAttnArgs a, int bt_shift) {
    using L = La<RANK, MT>;
    constexpr int CW = L::CW, PITCH = L::PITCH, KS = L::KS, NT = L::NT, HEADS = MT * 16;
    extern __shared__ __align__(16) unsigned char la_raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tq = lane & 3;
    __half* ring = reinterpret_cast<__half*>(la_raw) + warp * LA_STAGES * L::STAGE;
    float* scores = reinterpret_cast<float*>(la_raw + (size_t)LA_WARPS * LA_STAGES * L::STAGE * 2);
    const int col0 = warp * CW, head0 = blockIdx.y * HEADS;
    pdl_trigger();
    pdl_wait();
    const LatentEntry e = load_entry(a.entries, blockIdx.x);
    const int len = e.pos + 1;
    const int chunk = ((len + e.n_shares - 1) / e.n_shares + LA_KT - 1) / LA_KT * LA_KT;
    const int k_lo = e.share * chunk, k_hi = min(len, k_lo + chunk);
    const int tiles = k_hi > k_lo ? (k_hi - k_lo + LA_KT - 1) / LA_KT : 0;

    // the warp's columns of the queries, as A fragments
    uint32_t qf[MT][KS][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int k = 0; k < KS; ++k)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int head = head0 + m * 16 + gid + (i & 1) * 8, c = col0 + k * 16 + 2 * tq + (i >> 1) * 8;
                qf[m][k][i] = head < a.heads ? *reinterpret_cast<const uint32_t*>(a.q_h + ((int64_t)e.row * a.heads + head) * RANK + c) : 0u;
            }

    const __half* pool = static_cast<const __half*>(a.pool);
    auto row_of = [&](int t) {  // pool row of this lane's key of tile t
        const int pos = k_lo + t * LA_KT + lane;
        return pos < k_hi ? ((int64_t)a.tables[e.table_off + (pos >> bt_shift)] << bt_shift) + (pos & ((1 << bt_shift) - 1)) : (int64_t)-1;
    };
    constexpr int CHUNKS = CW / 8;  // 16-byte pieces of a row
    auto load = [&](int t, int64_t my_row) {
        __half* dst = ring + (t % LA_STAGES) * L::STAGE;
#pragma unroll
        for (int i = 0; i < CHUNKS; ++i) {
            const int j = i * 32 + lane, key = j / CHUNKS, c = (j % CHUNKS) * 8;
            const int64_t row = __shfl_sync(0xffffffffu, my_row, key);
            const int bytes = row >= 0 ? 16 : 0;  // keys past the end are zeros
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(la_smem(dst + key * PITCH + c)), "l"(pool + (row >= 0 ? row : 0) * RANK + col0 + c),
                         "r"(bytes)
                         : "memory");
        }
    };

    float o[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < NT; ++j) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.f;
    float m_run[MT][2], l_run[MT][2];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
        m_run[m][0] = m_run[m][1] = -INFINITY;
        l_run[m][0] = l_run[m][1] = 0.f;
    }

    int64_t next_row = 0;
    if (tiles > 0) load(0, row_of(0));
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (tiles > 1) next_row = row_of(1);
    for (int t = 0; t < tiles; ++t) {
        if (t + 1 < tiles) load(t + 1, next_row);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (t + 2 < tiles) next_row = row_of(t + 2);
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncwarp();
        const __half* rows = ring + (t % LA_STAGES) * L::STAGE;
        float* mine = scores + (t & 1) * L::SCORES;

        // this warp's part of the scores
        float s[MT][4][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int j = 0; j < 4; ++j) s[m][j][0] = s[m][j][1] = s[m][j][2] = s[m][j][3] = 0.f;
#pragma unroll
        for (int k = 0; k < KS; ++k)
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                uint32_t b[4];
                la_ldm4(b, rows + (j * 8 + (lane & 7) + (lane >> 4) * 8) * PITCH + k * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    la_mma(s[m][j], qf[m][k], b[0], b[1]);
                    la_mma(s[m][j + 1], qf[m][k], b[2], b[3]);
                }
            }
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h)
                    *reinterpret_cast<float2*>(mine + ((warp * MT + m) * 16 + gid + 8 * h) * LA_SP + j * 8 + 2 * tq) = make_float2(s[m][j][2 * h], s[m][j][2 * h + 1]);
        __syncthreads();
        const int pos0 = k_lo + t * LA_KT;
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    float2 v = make_float2(0.f, 0.f);
#pragma unroll
                    for (int w = 0; w < LA_WARPS; ++w) {
                        const float2 p = *reinterpret_cast<const float2*>(mine + ((w * MT + m) * 16 + gid + 8 * h) * LA_SP + j * 8 + 2 * tq);
                        v.x += p.x;
                        v.y += p.y;
                    }
                    const int pos = pos0 + j * 8 + 2 * tq;
                    s[m][j][2 * h] = pos < k_hi ? v.x * a.scale : -INFINITY;
                    s[m][j][2 * h + 1] = pos + 1 < k_hi ? v.y * a.scale : -INFINITY;
                    mx[h] = fmaxf(mx[h], fmaxf(s[m][j][2 * h], s[m][j][2 * h + 1]));
                }
            float alpha[2];
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
                mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
                const float m_new = fmaxf(m_run[m][h], mx[h]);  // finite: every tile has a visible key
                alpha[h] = __expf(m_run[m][h] - m_new);
                m_run[m][h] = m_new;
                float sum = 0.f;
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        const float p = __expf(s[m][j][2 * h + i] - m_new);
                        s[m][j][2 * h + i] = p;
                        sum += p;
                    }
                sum += __shfl_xor_sync(0xffffffffu, sum, 1);
                sum += __shfl_xor_sync(0xffffffffu, sum, 2);
                l_run[m][h] = l_run[m][h] * alpha[h] + sum;
            }
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                o[m][j][0] *= alpha[0];
                o[m][j][1] *= alpha[0];
                o[m][j][2] *= alpha[1];
                o[m][j][3] *= alpha[1];
            }
        }
#pragma unroll
        for (int kk = 0; kk < LA_KT / 16; ++kk) {
            uint32_t pf[MT][4], pr[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float x = s[m][2 * kk + (i >> 1)][(i & 1) * 2], y = s[m][2 * kk + (i >> 1)][(i & 1) * 2 + 1];
                    pf[m][i] = la_pack(x, y);
                    pr[m][i] = la_rest(x, y, pf[m][i]);
                }
#pragma unroll
            for (int j = 0; j < NT; j += 2) {
                uint32_t b[4];
                la_ldm4_trans(b, rows + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PITCH + j * 8 + (lane >> 4) * 8);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    la_mma(o[m][j], pf[m], b[0], b[1]);
                    la_mma(o[m][j + 1], pf[m], b[2], b[3]);
                    la_mma(o[m][j], pr[m], b[0], b[1]);
                    la_mma(o[m][j + 1], pr[m], b[2], b[3]);
                }
            }
        }
        __syncwarp();  // the stage is refilled by the next iteration's load
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");

    auto store = [&](int m, int h, int j, float x, float y, float f) {  // two neighbouring values of head row (m, h)
        const int head = head0 + m * 16 + gid + 8 * h;
        *reinterpret_cast<__nv_bfloat162*>(a.out.h + ((int64_t)head * a.n_rows + e.row) * RANK + col0 + j * 8 + 2 * tq) = __floats2bfloat162_rn(x * f, y * f);
    };
    if (e.n_shares == 1) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int head = head0 + m * 16 + gid + 8 * h;
                if (head >= a.heads) continue;
                const float f = sigmoid_f(a.gate.at(e.packed, a.gate_col + head)) / l_run[m][h];
#pragma unroll
                for (int j = 0; j < NT; ++j) store(m, h, j, o[m][j][2 * h], o[m][j][2 * h + 1], f);
            }
        return;
    }
    const int groups = gridDim.y;
    auto slot = [&](int entry) { return ((int64_t)entry * groups + blockIdx.y) * HEADS; };
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int item = m * 16 + gid + 8 * h;
            if (head0 + item >= a.heads) continue;
            float* po = a.part_o + (slot(blockIdx.x) + item) * RANK + col0;
#pragma unroll
            for (int j = 0; j < NT; ++j) *reinterpret_cast<float2*>(po + j * 8 + 2 * tq) = make_float2(o[m][j][2 * h], o[m][j][2 * h + 1]);
            if (warp == 0 && tq == 0) *reinterpret_cast<float2*>(a.part_ml + (slot(blockIdx.x) + item) * 2) = make_float2(m_run[m][h], l_run[m][h]);
        }
    __shared__ int s_last;
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        int32_t* counter = a.counters + (int64_t)e.first * groups + blockIdx.y;
        s_last = atomicAdd(counter, 1) == e.n_shares - 1 ? 1 : 0;
        if (s_last) *counter = 0;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
#pragma unroll 1
    for (int m = 0; m < MT; ++m)
#pragma unroll 1
        for (int h = 0; h < 2; ++h) {
            const int item = m * 16 + gid + 8 * h, head = head0 + item;
            if (head >= a.heads) continue;
            float mx = -INFINITY;
            for (int sh = 0; sh < e.n_shares; ++sh) mx = fmaxf(mx, __ldcg(a.part_ml + (slot(e.first + sh) + item) * 2));
            float l = 0.f, acc[NT][2];
#pragma unroll
            for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = 0.f;
            for (int sh = 0; sh < e.n_shares; ++sh) {
                const int64_t at = slot(e.first + sh) + item;
                const float2 ml = __ldcg(reinterpret_cast<const float2*>(a.part_ml + at * 2));
                if (ml.x == -INFINITY) continue;
                const float f = __expf(ml.x - mx);
                l += ml.y * f;
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    const float2 v = __ldcg(reinterpret_cast<const float2*>(a.part_o + at * RANK + col0 + j * 8 + 2 * tq));
                    acc[j][0] = fmaf(v.x, f, acc[j][0]);
                    acc[j][1] = fmaf(v.y, f, acc[j][1]);
                }
            }
            const float f = sigmoid_f(a.gate.at(e.packed, a.gate_col + head)) / l;
#pragma unroll
            for (int j = 0; j < NT; ++j) store(m, h, j, acc[j][0], acc[j][1], f);
        }
}

// ------------------------------------------------------------------------------------------------ general kernel

// f32 on the CUDA cores for f32 or f16 pages and any rank up to kLatentMaxRank: a CTA takes up to 16 heads of one query row, two
// per warp; tiles of 32 page rows are widened into shared memory, a lane scores one key and adds up every 32nd column.
constexpr int LG_WARPS = 8;
constexpr int LG_ITEMS = 2;
constexpr int LG_KEYS = 32;
constexpr int LG_COLS = kLatentMaxRank / 32;

template <typename KV>
__device__ __forceinline__ float la_widen(KV v);
template <>
__device__ __forceinline__ float la_widen<float>(float v) { return v; }
template <>
__device__ __forceinline__ float la_widen<__half>(__half v) { return __half2float(v); }

template <typename KV>
__global__ void __launch_bounds__(LG_WARPS * 32) latent_general_kernel(LatentAttnArgs a) {
    extern __shared__ __align__(16) float lg_smem[];
    const int R = a.rank, pitch = R + 4;
    float* qs = lg_smem;                              // [16][R]
    float* ks = qs + LG_WARPS * LG_ITEMS * R;         // [LG_KEYS][pitch]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    pdl_wait();
    const LatentEntry e = load_entry(a.entries, blockIdx.x);
    const int head0 = blockIdx.y * LG_WARPS * LG_ITEMS, heads = min(LG_WARPS * LG_ITEMS, a.heads - head0);
    const float* q = a.q_f + ((int64_t)e.row * a.heads + head0) * R;
    for (int i = threadIdx.x; i < heads * R; i += LG_WARPS * 32) qs[i] = q[i];
    float m_run[LG_ITEMS], l_run[LG_ITEMS], acc[LG_ITEMS][LG_COLS];
#pragma unroll
    for (int i = 0; i < LG_ITEMS; ++i) {
        m_run[i] = -INFINITY;
        l_run[i] = 0.f;
#pragma unroll
        for (int j = 0; j < LG_COLS; ++j) acc[i][j] = 0.f;
    }
    const KV* pool = static_cast<const KV*>(a.pool);
    for (int k0 = 0; k0 <= e.pos; k0 += LG_KEYS) {
        __syncthreads();
        for (int key = warp; key < LG_KEYS; key += LG_WARPS) {
            const int pos = k0 + key;
            if (pos <= e.pos) {
                const KV* src = pool + ((int64_t)a.tables[e.table_off + pos / a.block_tokens] * a.block_tokens + pos % a.block_tokens) * R;
                for (int c = lane; c < R; c += 32) ks[key * pitch + c] = la_widen<KV>(src[c]);
            } else {
                for (int c = lane; c < R; c += 32) ks[key * pitch + c] = 0.f;
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < LG_ITEMS; ++i) {
            const int item = warp + LG_WARPS * i;
            if (item >= heads) continue;
            const bool visible = k0 + lane <= e.pos;
            float s = -INFINITY;
            if (visible) {
                float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
                const float4* qv = reinterpret_cast<const float4*>(qs + item * R);
                const float4* kv = reinterpret_cast<const float4*>(ks + lane * pitch);
                for (int c = 0; c < R / 4; ++c) {
                    const float4 x = qv[c], y = kv[c];
                    d.x = fmaf(x.x, y.x, d.x);
                    d.y = fmaf(x.y, y.y, d.y);
                    d.z = fmaf(x.z, y.z, d.z);
                    d.w = fmaf(x.w, y.w, d.w);
                }
                s = (d.x + d.y + (d.z + d.w)) * a.scale;
            }
            const float m_new = fmaxf(m_run[i], warp_max(s));
            const float alpha = m_run[i] == -INFINITY ? 0.f : expf(m_run[i] - m_new);
            const float p = visible ? expf(s - m_new) : 0.f;
            l_run[i] = l_run[i] * alpha + warp_sum(p);
            m_run[i] = m_new;
#pragma unroll
            for (int j = 0; j < LG_COLS; ++j) acc[i][j] *= alpha;
            for (int key = 0; key < LG_KEYS; ++key) {
                const float pk = __shfl_sync(0xffffffffu, p, key);
                const float* v = ks + key * pitch + lane;
#pragma unroll
                for (int j = 0; j < LG_COLS; ++j)
                    if (j * 32 < R) acc[i][j] = fmaf(pk, v[j * 32], acc[i][j]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < LG_ITEMS; ++i) {
        const int item = warp + LG_WARPS * i;
        if (item >= heads) continue;
        const float f = sigmoid_f(a.gate.at(e.packed, a.gate_col + head0 + item)) / l_run[i];
#pragma unroll
        for (int j = 0; j < LG_COLS; ++j)
            if (j * 32 < R) a.out.put((int64_t)(head0 + item) * a.n_rows + e.row, j * 32 + lane, acc[i][j] * f);
    }
}

// ------------------------------------------------------------------------------------------------ rows in and out

__device__ __forceinline__ uint32_t la_bf2(float x, float y) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
    return *reinterpret_cast<const uint32_t*>(&v);
}

template <typename KV>
__global__ void __launch_bounds__(256) latent_gather_kernel(const KV* pool, const int32_t* blocks, int64_t rows, int block_tokens, int rank, __nv_bfloat16* out) {
    pdl_trigger();
    pdl_wait();
    const int per = rank / 8;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < rows * per; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = i / per;
        const int c = (int)(i - r * per) * 8;
        const KV* src = pool + ((int64_t)blocks[r / block_tokens] * block_tokens + r % block_tokens) * rank + c;
        KV v[8];
        *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(src);
        if (sizeof(KV) == 4) *reinterpret_cast<uint4*>(v + 4) = *reinterpret_cast<const uint4*>(src + 4);
        *reinterpret_cast<uint4*>(out + r * rank + c) =
            make_uint4(la_bf2(la_widen<KV>(v[0]), la_widen<KV>(v[1])), la_bf2(la_widen<KV>(v[2]), la_widen<KV>(v[3])),
                       la_bf2(la_widen<KV>(v[4]), la_widen<KV>(v[5])), la_bf2(la_widen<KV>(v[6]), la_widen<KV>(v[7])));
    }
}

__global__ void __launch_bounds__(256) split_rows_kernel(const float* x, int ldx, const int32_t* rows, int n_rows, int parts, int width, __nv_bfloat16* out) {
    pdl_trigger();
    pdl_wait();
    const float* src = x + (int64_t)rows[blockIdx.x] * ldx;
    for (int i = threadIdx.x * 4; i < parts * width; i += 1024) {  // width is a multiple of 64
        const int part = i / width, c = i - part * width;
        const float4 v = *reinterpret_cast<const float4*>(src + i);
        *reinterpret_cast<uint2*>(out + ((int64_t)part * n_rows + blockIdx.x) * width + c) = make_uint2(la_bf2(v.x, v.y), la_bf2(v.z, v.w));
    }
}

template <int RANK, int MT>
void launch_tc(const LatentAttnArgs& a, cudaStream_t s) {
    constexpr size_t smem = La<RANK, MT>::BYTES;
    int shift = 0;
    while ((1 << shift) < a.block_tokens) ++shift;
    ensure_dynamic_smem(reinterpret_cast<const void*>(&latent_tc_kernel<RANK, MT>), smem);
    launch_pdl(latent_tc_kernel<RANK, MT>, dim3((unsigned)a.n_entries, (unsigned)latent_tc_groups(a.heads)), dim3(LA_WARPS * 32), smem, s, a, shift);
}

template <int RANK>
void launch_tc_heads(const LatentAttnArgs& a, cudaStream_t s) {
    if (latent_tc_heads(a.heads) == 16) launch_tc<RANK, 1>(a, s);
    else launch_tc<RANK, 2>(a, s);
}

}  // namespace

int latent_tc_rank(int kv_rank, int block_tokens) {
    if (block_tokens <= 0 || (block_tokens & (block_tokens - 1)) != 0) return 0;
    for (int r : {64, 128, 256, 512})
        if (kv_rank <= r) return r;
    return 0;
}

int latent_tc_heads(int heads) { return heads <= 16 ? 16 : 32; }

int latent_max_shared_entries(int head_groups) { return std::max(LA_SHARED_ROWS + LA_SHARED_ROWS / 2, LA_TARGET_CTAS / head_groups) + 1; }
int latent_max_entries(int tokens, int head_groups) { return std::max(tokens, latent_max_shared_entries(head_groups)); }

void plan_latent_attention(const int32_t* start_pos, const int32_t* n_tokens, const int32_t* n_blocks, int lanes, int head_groups, int wide_from,
                           bool shares, LatentPlan& plan) {
    plan.entries.clear();
    plan.rows.clear();
    int rows = 0;
    int64_t keys = 0;
    for (int i = 0; i < lanes; ++i)
        if (n_tokens[i] < wide_from) {
            rows += n_tokens[i];
            keys += (int64_t)n_tokens[i] * start_pos[i] + (int64_t)n_tokens[i] * (n_tokens[i] + 1) / 2;
        }
    // Every CTA should walk about the same number of keys and all of them fit on the GPU at once.  Once the rows alone fill it, only
    // a row more than twice as long as the mean is cut.
    int share = 1 << 30;
    if (shares && rows > 0 && rows <= LA_SHARED_ROWS) {
        const bool filled = rows * head_groups >= LA_TARGET_CTAS;
        const int slots = filled ? rows + rows / 2 : std::max(rows, LA_TARGET_CTAS / head_groups);
        share = (int)std::max<int64_t>(LA_MIN_SHARE, filled ? 2 * (keys / rows) : (keys + slots - 1) / slots);
        for (;; share += LA_KT) {
            int64_t n = 0;
            for (int i = 0; i < lanes; ++i)
                if (n_tokens[i] < wide_from)
                    for (int t = 0; t < n_tokens[i]; ++t) n += std::min<int64_t>(LA_MAX_SHARES, (start_pos[i] + t + share) / share);
            if (n <= slots) break;
        }
    }
    int packed = 0, table_off = 0;
    for (int i = 0; i < lanes; packed += n_tokens[i], table_off += n_blocks[i], ++i) {
        if (n_tokens[i] >= wide_from) continue;
        for (int t = 0; t < n_tokens[i]; ++t) {
            const int pos = start_pos[i] + t, n = std::max(1, std::min(LA_MAX_SHARES, (int)(((int64_t)pos + share) / share)));
            const int first = plan.n_entries(), row = plan.n_rows();
            for (int k = 0; k < n; ++k)
                for (int32_t v : {row, k, n, pos, table_off, packed + t, first, 0}) plan.entries.push_back(v);
            plan.rows.push_back(packed + t);
        }
    }
}

void launch_latent_attention(const LatentAttnArgs& a, cudaStream_t s) {
    if (a.n_entries <= 0) return;
    if (a.out.ld != a.rank) throw std::runtime_error("launch_latent_attention: the output's rows are as wide as the latent");
    if (a.q_h != nullptr) {
        if (!a.pool_f16 || a.out.h == nullptr) throw std::runtime_error("launch_latent_attention: f16 queries go with f16 pages and a bf16 output");
        switch (a.rank) {
            case 64: launch_tc_heads<64>(a, s); break;
            case 128: launch_tc_heads<128>(a, s); break;
            case 256: launch_tc_heads<256>(a, s); break;
            case 512: launch_tc_heads<512>(a, s); break;
            default: throw std::runtime_error("launch_latent_attention: unsupported rank");
        }
    } else {
        if (a.rank % 32 != 0 || a.rank > kLatentMaxRank) throw std::runtime_error("launch_latent_attention: latents above 1024 values are not supported");
        const size_t smem = ((size_t)LG_WARPS * LG_ITEMS * a.rank + (size_t)LG_KEYS * (a.rank + 4)) * 4;
        auto* kernel = a.pool_f16 ? latent_general_kernel<__half> : latent_general_kernel<float>;
        const dim3 grid((unsigned)a.n_entries, (unsigned)((a.heads + LG_WARPS * LG_ITEMS - 1) / (LG_WARPS * LG_ITEMS)));
        ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), smem);
        launch_pdl(kernel, grid, dim3(LG_WARPS * 32), smem, s, a);
    }
    MK_LAUNCH_CHECK();
}

void launch_latent_gather(const void* pool, int pool_f16, const int32_t* blocks, int n_blocks, int block_tokens, int rank, __nv_bfloat16* out, cudaStream_t s) {
    if (n_blocks <= 0) return;
    if (rank % 8 != 0) throw std::runtime_error("launch_latent_gather: the rank must be a multiple of 8");
    const int64_t rows = (int64_t)n_blocks * block_tokens;
    const dim3 grid((unsigned)std::min<int64_t>((rows * (rank / 8) + 255) / 256, LA_SMS * 16));
    if (pool_f16) launch_pdl(latent_gather_kernel<__half>, grid, dim3(256), 0, s, static_cast<const __half*>(pool), blocks, rows, block_tokens, rank, out);
    else launch_pdl(latent_gather_kernel<float>, grid, dim3(256), 0, s, static_cast<const float*>(pool), blocks, rows, block_tokens, rank, out);
    MK_LAUNCH_CHECK();
}

void launch_split_rows(const float* x, int ldx, const int32_t* rows, int n_rows, int parts, int width, __nv_bfloat16* out, cudaStream_t s) {
    if (n_rows <= 0) return;
    if (width % 4 != 0 || ldx % 4 != 0) throw std::runtime_error("launch_split_rows: widths must be multiples of 4");
    launch_pdl(split_rows_kernel, dim3((unsigned)n_rows), dim3(256), 0, s, x, ldx, rows, n_rows, parts, width, out);
    MK_LAUNCH_CHECK();
}

}  // namespace mk
