// See latent_attention.h.
//
// Tensor-core kernel (tcgen05): one CTA per (query row, share of its keys, up to 32 heads).  Tiles of 128 cached vectors arrive in
// chunks of 128 columns as 128-byte swizzled rows, by 16-byte cp.async (TMA boxes as small as a page's part of a chunk brought
// them no faster).  A tile is an operand twice: with the vectors' columns as the reduction it gives the scores transposed (keys x
// heads), and read the other way round, with the keys as the reduction, it gives the outputs transposed (columns x heads) - so the
// wide side of both products fills the tensor core's 128 rows and the few heads are its columns.  Four groups of four warps, a
// quarter of the heads each, hold one key per thread: scores from tensor memory, the heads' maxima over the keys by a folding
// exchange, softmax weights in f32, which go back to shared memory as two f16 numbers each (high part and rest, as columns of
// their own, added up at the end).  The MMA issuer takes what is ready first, the weights of a tile or the next chunk of the tile
// after it, so scores go ahead of outputs as far as the ring holds them.  The running maximum moves only when a tile exceeds it by
// more than kSlack, so the accumulators in tensor memory are hardly ever rescaled.  When few rows are in flight their keys are
// shared out over several CTAs; the one that finishes last adds the shares in order.  Every wait is bounded (see hgemm_tc.cu).
#include "latent_attention.h"
#include "kernels.h"
#include "device_util.h"
#include <algorithm>

namespace mk {

namespace {

constexpr int LU_KEYS = 128;          // keys of a tile
constexpr int LU_COLS = 128;          // columns of a chunk
constexpr int LU_CHUNK = LU_KEYS * LU_COLS * 2;
constexpr int LU_BLOCK = LU_KEYS * 128;  // bytes of the 64 columns that share swizzled rows
constexpr int LU_GROUPS = 4;           // softmax groups of four warps
constexpr int LU_SOFTMAX = LU_GROUPS * 128;
constexpr int LU_LOADERS = 128;
constexpr int LU_THREADS = LU_SOFTMAX + LU_LOADERS + 32;  // and the MMA issuer's warp
constexpr float kSlack = 8.f;         // weights stay below e^8, well inside f16
constexpr uint32_t LU_SPIN_LIMIT = 1u << 22;
constexpr int LA_SMS = 148;
constexpr int LA_TARGET_CTAS = LA_SMS;
constexpr int LA_MIN_SHARE = 256;
constexpr int LA_MAX_SHARES = 32;
constexpr int LA_SHARED_ROWS = 256;   // ticks with more query rows are not cut into shares

__device__ __forceinline__ uint32_t lu_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void lu_bar_init(uint64_t* bar, uint32_t count) { asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(lu_smem(bar)), "r"(count)); }
__device__ __forceinline__ bool lu_bar_wait(uint64_t* bar, uint32_t parity) {
    const uint32_t addr = lu_smem(bar);
    for (uint32_t i = 0; i <= LU_SPIN_LIMIT; ++i) {
        uint32_t done;
        asm volatile(
            "{\n\t.reg .pred p;\n\t"
            "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
            "selp.u32 %0, 1, 0, p;\n\t}"
            : "=r"(done)
            : "r"(addr), "r"(parity)
            : "memory");
        if (done) return true;
    }
    return false;
}
__device__ __forceinline__ bool lu_bar_test(uint64_t* bar, uint32_t parity) {
    uint32_t done;
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(done)
        : "r"(lu_smem(bar)), "r"(parity)
        : "memory");
    return done != 0;
}
__device__ __forceinline__ void lu_bar_arrive(uint64_t* bar) { asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(lu_smem(bar)) : "memory"); }
// 16 bytes (zeros when there is no source), counted on the barrier together with the thread's other copies by lu_copies_arrive.
__device__ __forceinline__ void lu_copy16(uint32_t dst, const void* src, bool valid) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void lu_copies_arrive(uint64_t* bar) {
    asm volatile("cp.async.mbarrier.arrive.noinc.shared::cta.b64 [%0];" ::"r"(lu_smem(bar)) : "memory");
}
// Operand of 128-byte swizzled rows, 8-row groups 1024 bytes apart.  Reduction along the rows' bytes: lead is not used; reduction
// from row to row: lead = distance of the next 64 elements of the other dimension.
__device__ __forceinline__ uint64_t lu_desc(uint32_t addr, uint32_t lead) {
    return (uint64_t)((addr >> 4) & 0x3FFF) | (uint64_t)(lead >> 4) << 16 | (uint64_t)(1024 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)2 << 61;
}
__device__ __forceinline__ void lu_mma(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, bool accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(d), "l"(a), "l"(b), "r"(idesc), "r"(accumulate ? 1u : 0u)
        : "memory");
}
__device__ __forceinline__ void lu_commit(uint64_t* bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(lu_smem(bar)) : "memory");
}
// N (4 or 8) columns of this thread's lane; the values are there after lu_tmem_wait.
template <int N>
__device__ __forceinline__ void lu_tmem_load(uint32_t at, uint32_t* r) {
    if constexpr (N == 4)
        asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at) : "memory");
    else
        asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                     : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                     : "r"(at)
                     : "memory");
}
template <int N>
__device__ __forceinline__ void lu_tmem_store(uint32_t at, const uint32_t* r) {
    if constexpr (N == 4)
        asm volatile("tcgen05.st.sync.aligned.32x32b.x4.b32 [%0], {%1,%2,%3,%4};" ::"r"(at), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]) : "memory");
    else
        asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"r"(at), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]),
                     "r"(r[6]), "r"(r[7])
                     : "memory");
}
__device__ __forceinline__ void lu_tmem_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void lu_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void lu_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
// Barrier of `threads` softmax threads; true when every one of them came with ok.
__device__ __forceinline__ bool lu_agree(int barrier, int threads, bool ok) {
    uint32_t all;
    asm volatile(
        "{\n\t.reg .pred p, q;\n\t"
        "setp.ne.u32 q, %1, 0;\n\t"
        "bar.red.and.pred p, %2, %3, q;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(all)
        : "r"(ok ? 1u : 0u), "r"(barrier), "r"(threads)
        : "memory");
    return all != 0;
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
// N values per lane, folded over the warp: lane l ends with the result of value l % N over all lanes.  Uses up v.
template <int N, typename Op>
__device__ __forceinline__ float lu_fold(float (&v)[N], int lane, Op op) {
#pragma unroll
    for (int s = N / 2; s > 0; s >>= 1) {
        const bool up = (lane & s) != 0;
#pragma unroll
        for (int i = 0; i < N / 2; ++i)
            if (i < s) v[i] = op(up ? v[i + s] : v[i], __shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + s], s));
    }
    float r = v[0];
#pragma unroll
    for (int s = N; s < 32; s <<= 1) r = op(r, __shfl_xor_sync(0xffffffffu, r, s));
    return r;
}

struct LatentEntry {
    int row, share, n_shares, pos, table_off, packed, first;
};
__device__ __forceinline__ LatentEntry load_entry(const int32_t* entries, int i) {
    const int4 a = reinterpret_cast<const int4*>(entries)[2 * i], b = reinterpret_cast<const int4*>(entries)[2 * i + 1];
    return LatentEntry{a.x, a.y, a.z, a.w, b.x, b.y, b.z};
}

// What the softmax's denominator, exp(m) l without it, is with one more term exp(sink): exp(m) times the result.
__device__ __forceinline__ float la_with_sink(const float* sink, int head, float m, float l) {
    return sink == nullptr ? l : l + __expf(fminf(sink[head] - m, 80.f));
}
// Two neighbouring query columns at `turn` of the rotation tables.
__device__ __forceinline__ float2 la_turn(float2 v, const LatentAttnArgs& a, int64_t turn) {
    const float cs = a.cos_t[turn], sn = a.sin_t[turn];
    return make_float2(v.x * cs - v.y * sn, v.y * cs + v.x * sn);
}

// MB chunks of 128 value columns, then XB blocks of 64 columns that count in the scores only; NH heads (16 or 32).
template <int MB, int NH, int XB>
struct Lu {
    static constexpr int VALUES = MB * LU_COLS, RANK = VALUES + XB * 64;
    static constexpr int CHUNKS = MB + (XB > 0 ? 1 : 0);   // of a tile; the last one may be half as wide
    static constexpr int BASE = MB >= 4 && NH == 16 ? 6 : (MB >= 3 ? 5 : (MB == 2 ? 4 : 2));
    static constexpr int STAGES = XB > 0 && MB == 1 ? 4 : BASE;                                 // chunks in the ring
    static constexpr int Q_BYTES = NH * RANK * 2;                                               // [column block][head][64]
    static constexpr int P_BYTES = 2 * NH * LU_KEYS * 2;                                        // [key block][weights | rests][64]
    static constexpr size_t BYTES = (size_t)STAGES * LU_CHUNK + Q_BYTES + P_BYTES + 1024 + 256;
    static constexpr int S_COL = MB * 2 * NH;  // tensor memory: outputs (high | rest) of every chunk, then two tiles' scores
    static constexpr int END_COL = S_COL + 2 * NH;
    static constexpr uint32_t TMEM = END_COL <= 64 ? 64 : END_COL <= 128 ? 128 : (END_COL <= 256 ? 256 : 512);
    static_assert(END_COL <= 512 && STAGES >= CHUNKS, "tensor memory; a tile fits in the ring");
};

template <int MB, int NH, int XB>
__global__ void __launch_bounds__(LU_THREADS, 1) latent_umma_kernel(LatentAttnArgs a, int bt_shift) {
    using L = Lu<MB, NH, XB>;
    constexpr int RANK = L::RANK, VALUES = L::VALUES, CHUNKS = L::CHUNKS, STAGES = L::STAGES, HG = NH / LU_GROUPS, LOADER = LU_SOFTMAX / 32;
    extern __shared__ uint8_t lu_raw[];
    uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lu_raw) + 1023) & ~(uintptr_t)1023);
    uint8_t* qs = ring + (size_t)STAGES * LU_CHUNK;
    uint8_t* ps = qs + L::Q_BYTES;
    uint64_t* full = reinterpret_cast<uint64_t*>(ps + L::P_BYTES);  // [STAGES] loader -> MMA
    uint64_t* empty = full + STAGES;                                // [STAGES] MMA -> loader
    uint64_t* q_full = empty + STAGES;                              // softmax -> MMA: queries
    uint64_t* s_full = q_full + 1;                                  // [2] MMA -> softmax: scores
    uint64_t* p_full = s_full + 2;                                  // softmax -> MMA: weights
    uint64_t* o_done = p_full + 1;                                  // MMA -> softmax: the tile is in the outputs
    __shared__ uint32_t tmem_slot;
    __shared__ __align__(16) float s_warp[LU_SOFTMAX / 32][HG], s_factor[LA_MAX_SHARES][NH];
    __shared__ int s_last, s_rows[2][LU_KEYS];

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int head0 = blockIdx.y * NH, heads = min(NH, a.heads - head0);
    if (tid == 0) {
        for (int i = 0; i < STAGES; ++i) {
            lu_bar_init(&full[i], LU_LOADERS);
            lu_bar_init(&empty[i], 1);
        }
        lu_bar_init(q_full, LU_SOFTMAX);
        lu_bar_init(&s_full[0], 1);
        lu_bar_init(&s_full[1], 1);
        lu_bar_init(p_full, LU_SOFTMAX);
        lu_bar_init(o_done, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == LOADER) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(lu_smem(&tmem_slot)), "r"(L::TMEM) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    lu_fence_before();
    __syncthreads();
    lu_fence_after();
    const uint32_t tmem = tmem_slot;
    pdl_trigger();
    // work list and block tables were staged by the host: they need not wait for the predecessor
    const LatentEntry e = load_entry(a.entries, blockIdx.x);
    const int first_key = attention_first_key(e.pos, a.window, 0), len = e.pos + 1 - first_key;
    const int chunk = ((len + e.n_shares - 1) / e.n_shares + LU_KEYS - 1) / LU_KEYS * LU_KEYS;
    const int k_lo = first_key + e.share * chunk, k_hi = min(e.pos + 1, k_lo + chunk);
    const int tiles = k_hi > k_lo ? (k_hi - k_lo + LU_KEYS - 1) / LU_KEYS : 0;
    auto row_of = [&](int t, int key) {  // pool row of a tile's key, -1 past the last one
        const int pos = k_lo + t * LU_KEYS + key;
        return pos < k_hi ? (int)(a.tables[e.table_off + (pos >> bt_shift)] << bt_shift) + (pos & ((1 << bt_shift) - 1)) : -1;
    };
    if (warp >= LOADER && warp < LOADER + LU_LOADERS / 32 && tiles > 0) s_rows[0][tid - LU_SOFTMAX] = row_of(0, tid - LU_SOFTMAX);
    pdl_wait();

    if (warp >= LOADER && warp < LOADER + LU_LOADERS / 32) {
        // ---- loaders: pool rows of a tile's keys first (one per thread), then 16-byte pieces of the rows
        static_assert(LU_LOADERS == LU_KEYS, "a loader thread looks up one key");
        const int lt = tid - LU_SOFTMAX, piece = lt & 15, key0 = lt >> 4;
        const __half* pool = static_cast<const __half*>(a.pool) + piece * 8;
        const uint32_t dst0 = lu_smem(ring) + (piece >> 3) * LU_BLOCK;
        uint32_t it = 0;
        bool ok = true;
        for (int t = 0; t < tiles; ++t) {
            ok = lu_agree(LU_GROUPS + 2, LU_LOADERS, ok);  // this tile's rows are there, nobody reads the other buffer any more
            if (!ok) break;
            if (t + 1 < tiles) s_rows[(t + 1) & 1][lt] = row_of(t + 1, lt);
            for (int c = 0; c < CHUNKS; ++c, ++it) {
                const uint32_t st = it % STAGES;
                ok = lu_bar_wait(&empty[st], ((it / STAGES) & 1) ^ 1);
                if (!ok) break;
                if (XB == 1 && c == MB && piece >= 8) {  // half a chunk
                    lu_copies_arrive(&full[st]);
                    continue;
                }
                const uint32_t dst = dst0 + st * LU_CHUNK;
                const __half* src = pool + c * LU_COLS;
#pragma unroll
                for (int j = 0; j < LU_KEYS / 8; ++j) {
                    const int key = j * 8 + key0, row = s_rows[t & 1][key];
                    lu_copy16(dst + key * 128 + (((piece & 7) ^ (key & 7)) << 4), src + (int64_t)max(row, 0) * RANK, row >= 0);
                }
                lu_copies_arrive(&full[st]);
            }
        }
        if (!ok) atomicExch(a.status, 21);
        asm volatile("cp.async.wait_all;" ::: "memory");
    } else if (warp == LOADER + LU_LOADERS / 32) {
        // ---- MMA issuer
        if (lane == 0 && tiles > 0) {
            const uint32_t i_scores = (1u << 4) | ((uint32_t)(NH >> 3) << 17) | (8u << 24);
            const uint32_t i_out = (1u << 4) | (1u << 15) | ((uint32_t)(2 * NH >> 3) << 17) | (8u << 24);  // A read with the keys as the reduction
            const uint32_t q_addr = lu_smem(qs), p_addr = lu_smem(ps), ring_addr = lu_smem(ring);
            bool ok = true;
            auto scores = [&](int t, int c) {  // chunk c of tile t's scores; the chunk is there
                const uint32_t st = (uint32_t)(t * CHUNKS + c) % STAGES;
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // the copies are ordinary writes
                lu_fence_after();
                // descriptors hold addresses in 16-byte units
                const uint64_t keys = lu_desc(ring_addr + st * LU_CHUNK, 16), queries = lu_desc(q_addr + 2 * c * (NH * 128), 16);
                const uint32_t d = tmem + L::S_COL + (t & 1) * NH;
#pragma unroll
                for (int k = 0; k < LU_COLS / 16; ++k) {
                    if (XB == 1 && k >= 4 && c == MB) break;
                    lu_mma(d, keys + (k >> 2) * (LU_BLOCK / 16) + (k & 3) * 2, queries + (k >> 2) * (NH * 8) + (k & 3) * 2, i_scores, c > 0 || k > 0);
                }
                if (XB > 0 && c == MB) lu_commit(&empty[st]);  // nothing else reads it
                if (c == CHUNKS - 1) lu_commit(&s_full[t & 1]);
            };
            auto outputs = [&](int t) {  // tile t's part of the outputs; the weights are there
                lu_fence_after();
                const uint64_t weights = lu_desc(p_addr, 16);
                for (int c = 0; c < MB; ++c) {
                    const uint32_t st = (uint32_t)(t * CHUNKS + c) % STAGES;
                    const uint64_t values = lu_desc(ring_addr + st * LU_CHUNK, LU_BLOCK);
#pragma unroll
                    for (int k = 0; k < LU_KEYS / 16; ++k)
                        lu_mma(tmem + c * 2 * NH, values + k * 128, weights + (k >> 2) * (2 * NH * 8) + (k & 3) * 2, i_out, t > 0 || k > 0);
                    lu_commit(&empty[st]);
                }
                lu_commit(o_done);
            };
            auto full_of = [&](int t, int c) { return &full[(uint32_t)(t * CHUNKS + c) % STAGES]; };
            auto full_parity = [&](int t, int c) { return ((uint32_t)(t * CHUNKS + c) / STAGES) & 1; };
            ok = lu_bar_wait(q_full, 0);
            lu_fence_after();
            for (int c = 0; c < CHUNKS && ok; ++c) {
                ok = lu_bar_wait(full_of(0, c), full_parity(0, c));
                if (ok) scores(0, c);
            }
            // From here on whatever is ready first: the weights of tile t, or the next chunk of tile t + 1.  Chunks that find no room
            // beside tile t come only after its outputs.
            for (int t = 0; t < tiles && ok; ++t) {
                bool summed = false;
                int c = t + 1 < tiles ? 0 : CHUNKS;
                for (uint32_t spins = 0; ok && (!summed || c < CHUNKS);) {
                    if (!summed && lu_bar_test(p_full, t & 1)) {
                        outputs(t);
                        summed = true;
                        spins = 0;
                    }
                    if (c < CHUNKS && lu_bar_test(full_of(t + 1, c), full_parity(t + 1, c))) {
                        scores(t + 1, c);
                        ++c;
                        spins = 0;
                    }
                    ok = ++spins < LU_SPIN_LIMIT;
                }
            }
            if (!ok) atomicExch(a.status, 22);
        }
    } else {
        // ---- softmax: a group of 128 threads takes HG heads; thread = key of the tile, later column of a chunk
        const int group = warp >> 2, gt = tid & 127, h0 = group * HG, bar = 1 + group;
        // the queries, a head per row, 16-byte pieces
#pragma unroll 4
        for (int i = tid; i < NH * (RANK / 8); i += LU_SOFTMAX) {
            const int h = i / (RANK / 8), c = i - h * (RANK / 8);
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (h < heads) v = *reinterpret_cast<const uint4*>(a.q_h + ((int64_t)e.row * a.heads + head0 + h) * RANK + c * 8);
            const int turned = c * 8 - a.rot0;
            if (turned >= 0 && turned < a.rot_dims) {
                uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    if (turned + 2 * i >= a.rot_dims) break;
                    const float2 x = la_turn(__half22float2(*reinterpret_cast<const __half2*>(&w[i])), a, (int64_t)e.pos * (a.rot_dims / 2) + turned / 2 + i);
                    w[i] = la_pack(x.x, x.y);
                }
                v = make_uint4(w[0], w[1], w[2], w[3]);
            }
            *reinterpret_cast<uint4*>(qs + (c >> 3) * (NH * 128) + h * 128 + (((c & 7) ^ (h & 7)) << 4)) = v;
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        lu_bar_arrive(q_full);

        const uint32_t my_tmem = tmem + ((uint32_t)((warp & 3) * 32) << 16) + h0;
        float m[HG], l[HG];
#pragma unroll
        for (int h = 0; h < HG; ++h) {
            m[h] = -INFINITY;
            l[h] = 0.f;
        }
        bool ok = true;
        for (int t = 0; t < tiles; ++t) {
            ok = ok && lu_bar_wait(&s_full[t & 1], (t >> 1) & 1);
            __syncwarp();
            lu_fence_after();
            const bool visible = k_lo + t * LU_KEYS + gt < k_hi;
            uint32_t raw[HG];
            float s[HG], x[HG];
            lu_tmem_load<HG>(my_tmem + L::S_COL + (t & 1) * NH, raw);
            lu_tmem_wait();
#pragma unroll
            for (int h = 0; h < HG; ++h) x[h] = s[h] = visible ? __uint_as_float(raw[h]) * a.scale : -INFINITY;
            const float top = lu_fold<HG>(x, lane, [](float p, float q) { return fmaxf(p, q); });
            if (lane < HG) s_warp[warp][lane] = top;
            ok = lu_agree(bar, 128, ok);
            if (!ok) {
                if (gt == 0) atomicExch(a.status, 24);
                break;
            }
            bool moved = false;
            float keep[HG];
#pragma unroll
            for (int h = 0; h < HG; h += 4) {
                float4 v = *reinterpret_cast<const float4*>(&s_warp[group * 4][h]);
#pragma unroll
                for (int w = 1; w < 4; ++w) {
                    const float4 u = *reinterpret_cast<const float4*>(&s_warp[group * 4 + w][h]);
                    v = make_float4(fmaxf(v.x, u.x), fmaxf(v.y, u.y), fmaxf(v.z, u.z), fmaxf(v.w, u.w));
                }
                const float tile_max[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    keep[h + i] = 1.f;
                    if (t == 0 || tile_max[i] > m[h + i] + kSlack) {  // the same in every thread
                        keep[h + i] = t == 0 ? 0.f : __expf(m[h + i] - tile_max[i]);
                        m[h + i] = tile_max[i];
                        moved = true;
                    }
                }
            }
            // weights and rests of two heads at a time
            uint32_t hi[HG / 2], lo[HG / 2];
#pragma unroll
            for (int h = 0; h < HG; h += 2) {
                const float p0 = visible ? __expf(s[h] - m[h]) : 0.f, p1 = visible ? __expf(s[h + 1] - m[h + 1]) : 0.f;
                l[h] = fmaf(l[h], keep[h], p0);
                l[h + 1] = fmaf(l[h + 1], keep[h + 1], p1);
                hi[h / 2] = la_pack(p0, p1);
                lo[h / 2] = la_rest(p0, p1, hi[h / 2]);
            }
            if (t > 0) {
                ok = lu_bar_wait(o_done, (t - 1) & 1);  // the weights' buffer is free and the outputs stand still
                __syncwarp();
                lu_fence_after();
                if (moved) {
#pragma unroll 1
                    for (int c = 0; c < MB * 2; ++c) {
                        lu_tmem_load<HG>(my_tmem + c * NH, raw);
                        lu_tmem_wait();
#pragma unroll
                        for (int h = 0; h < HG; ++h) raw[h] = __float_as_uint(__uint_as_float(raw[h]) * keep[h]);
                        lu_tmem_store<HG>(my_tmem + c * NH, raw);
                    }
                    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
                }
            }
            uint8_t* col = ps + (gt >> 6) * (2 * NH * 128) + h0 * 128 + (gt & 7) * 2;
            const int piece = (gt & 63) >> 3;
#pragma unroll
            for (int h = 0; h < HG; ++h) {
                const int at = h * 128 + ((piece ^ ((h0 + h) & 7)) << 4);
                *reinterpret_cast<uint16_t*>(col + at) = (uint16_t)(h & 1 ? hi[h / 2] >> 16 : hi[h / 2]);
                *reinterpret_cast<uint16_t*>(col + NH * 128 + at) = (uint16_t)(h & 1 ? lo[h / 2] >> 16 : lo[h / 2]);
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            lu_fence_before();
            lu_bar_arrive(p_full);
        }
        if (ok && tiles > 0) ok = lu_bar_wait(o_done, (tiles - 1) & 1);
        __syncwarp();
        lu_fence_after();
        const float sum = lu_fold<HG>(l, lane, [](float p, float q) { return p + q; });
        lu_agree(bar, 128, true);  // the maxima have been read
        if (lane < HG) s_warp[warp][lane] = sum;
        if (!lu_agree(bar, 128, ok) && gt == 0) atomicExch(a.status, 25);
        auto slot = [&](int entry) { return ((int64_t)entry * gridDim.y + blockIdx.y) * NH; };
        auto gate_of = [&](int h) { return a.gate.p != nullptr ? sigmoid_f(a.gate.at(e.packed, a.gate_col + head0 + h)) : 1.f; };
        auto ml_at = [&](int entry, int h) { return a.part_ml + (slot(entry) + h) * 2; };
        if (gt < HG && h0 + gt < heads) {  // thread gt finishes head h0 + gt
            float total = 0.f, mine = -INFINITY;
#pragma unroll
            for (int w = 0; w < 4; ++w) total += s_warp[group * 4 + w][gt];
#pragma unroll
            for (int h = 0; h < HG; ++h)
                if (h == gt) mine = m[h];
            if (e.n_shares == 1) s_factor[0][h0 + gt] = gate_of(h0 + gt) / la_with_sink(a.sink, head0 + h0 + gt, mine, total);
            else *reinterpret_cast<float2*>(ml_at(blockIdx.x, h0 + gt)) = make_float2(mine, total);
        }
        lu_agree(bar, 128, true);
#pragma unroll
        for (int c = 0; c < MB; ++c) {
            uint32_t o[HG], rest[HG];
            if (tiles > 0) {
                lu_tmem_load<HG>(my_tmem + c * 2 * NH, o);
                lu_tmem_load<HG>(my_tmem + c * 2 * NH + NH, rest);
                lu_tmem_wait();
            }
#pragma unroll
            for (int h = 0; h < HG; ++h) {
                if (h0 + h >= heads) continue;
                const float v = tiles > 0 ? __uint_as_float(o[h]) + __uint_as_float(rest[h]) : 0.f;
                if (e.n_shares == 1)
                    a.out.h[((int64_t)(head0 + h0 + h) * a.n_rows + e.row) * VALUES + c * LU_COLS + gt] = __float2bfloat16_rn(v * s_factor[0][h0 + h]);
                else
                    a.part_o[(slot(blockIdx.x) + h0 + h) * VALUES + c * LU_COLS + gt] = v;
            }
        }
        if (e.n_shares > 1) {
            __threadfence();
            lu_agree(LU_GROUPS + 1, LU_SOFTMAX, true);
            if (tid == 0) {
                int32_t* counter = a.counters + (int64_t)e.first * gridDim.y + blockIdx.y;
                s_last = atomicAdd(counter, 1) == e.n_shares - 1 ? 1 : 0;
                if (s_last) *counter = 0;
            }
            lu_agree(LU_GROUPS + 1, LU_SOFTMAX, true);
            if (s_last) {
                __threadfence();
                if (tid < heads) {  // what every share of head `tid` is multiplied by
                    float mx = -INFINITY, total = 0.f;
                    for (int sh = 0; sh < e.n_shares; ++sh) mx = fmaxf(mx, __ldcg(ml_at(e.first + sh, tid)));
                    for (int sh = 0; sh < e.n_shares; ++sh) {
                        const float2 ml = __ldcg(reinterpret_cast<const float2*>(ml_at(e.first + sh, tid)));
                        const float f = ml.x == -INFINITY ? 0.f : __expf(ml.x - mx);
                        s_factor[sh][tid] = f;
                        total = fmaf(ml.y, f, total);
                    }
                    const float g = gate_of(tid) / la_with_sink(a.sink, head0 + tid, mx, total);
                    for (int sh = 0; sh < e.n_shares; ++sh) s_factor[sh][tid] *= g;
                }
                lu_agree(LU_GROUPS + 1, LU_SOFTMAX, true);
#pragma unroll 4
                for (int i = tid; i < heads * (MB * LU_COLS / 4); i += LU_SOFTMAX) {
                    const int h = i / (MB * LU_COLS / 4), c = (i - h * (MB * LU_COLS / 4)) * 4;
                    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
                    for (int sh = 0; sh < e.n_shares; ++sh) {
                        const float4 v = __ldcg(reinterpret_cast<const float4*>(a.part_o + (slot(e.first + sh) + h) * VALUES + c));
                        const float f = s_factor[sh][h];
                        acc = make_float4(fmaf(v.x, f, acc.x), fmaf(v.y, f, acc.y), fmaf(v.z, f, acc.z), fmaf(v.w, f, acc.w));
                    }
                    a.out.put4((int64_t)(head0 + h) * a.n_rows + e.row, c, acc);
                }
            }
        }
    }
    lu_fence_before();
    __syncthreads();
    if (warp == LOADER) {
        lu_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(L::TMEM) : "memory");
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
    const int R = a.rank, V = a.values, pitch = R + 4;
    float* qs = lg_smem;                              // [16][R]
    float* ks = qs + LG_WARPS * LG_ITEMS * R;         // [LG_KEYS][pitch]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    pdl_wait();
    const LatentEntry e = load_entry(a.entries, blockIdx.x);
    const int head0 = blockIdx.y * LG_WARPS * LG_ITEMS, heads = min(LG_WARPS * LG_ITEMS, a.heads - head0);
    const float* q = a.q_f + ((int64_t)e.row * a.heads + head0) * R;
    for (int i = threadIdx.x * 2; i < heads * R; i += LG_WARPS * 64) {
        float2 x = *reinterpret_cast<const float2*>(q + i);
        const int c = i % R - a.rot0;
        if (c >= 0 && c < a.rot_dims) x = la_turn(x, a, (int64_t)e.pos * (a.rot_dims / 2) + c / 2);
        *reinterpret_cast<float2*>(qs + i) = x;
    }
    const int first_key = attention_first_key(e.pos, a.window, 0);
    float m_run[LG_ITEMS], l_run[LG_ITEMS], acc[LG_ITEMS][LG_COLS];
#pragma unroll
    for (int i = 0; i < LG_ITEMS; ++i) {
        m_run[i] = -INFINITY;
        l_run[i] = 0.f;
#pragma unroll
        for (int j = 0; j < LG_COLS; ++j) acc[i][j] = 0.f;
    }
    const KV* pool = static_cast<const KV*>(a.pool);
    for (int k0 = first_key; k0 <= e.pos; k0 += LG_KEYS) {
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
                    if (j * 32 < V) acc[i][j] = fmaf(pk, v[j * 32], acc[i][j]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < LG_ITEMS; ++i) {
        const int item = warp + LG_WARPS * i;
        if (item >= heads) continue;
        const float gate = a.gate.p != nullptr ? sigmoid_f(a.gate.at(e.packed, a.gate_col + head0 + item)) : 1.f;
        const float f = gate / (a.sink != nullptr ? l_run[i] + expf(fminf(a.sink[head0 + item] - m_run[i], 80.f)) : l_run[i]);
#pragma unroll
        for (int j = 0; j < LG_COLS; ++j)
            if (j * 32 < V) a.out.put((int64_t)(head0 + item) * a.n_rows + e.row, j * 32 + lane, acc[i][j] * f);
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

template <int MB, int NH, int XB>
void launch_umma(const LatentAttnArgs& a, cudaStream_t s) {
    constexpr size_t smem = Lu<MB, NH, XB>::BYTES;
    static_assert(smem <= (size_t)227 * 1024, "shared memory");
    int shift = 0;
    while ((1 << shift) < a.block_tokens) ++shift;
    ensure_dynamic_smem(reinterpret_cast<const void*>(&latent_umma_kernel<MB, NH, XB>), smem);
    launch_pdl(latent_umma_kernel<MB, NH, XB>, dim3((unsigned)a.n_entries, (unsigned)latent_tc_groups(a.heads)), dim3(LU_THREADS), smem, s, a, shift);
}

template <int MB, int NH>
void launch_umma_extra(const LatentAttnArgs& a, cudaStream_t s) {
    switch (a.rank - a.values) {
        case 0: launch_umma<MB, NH, 0>(a, s); break;
        case 64: launch_umma<MB, NH, 1>(a, s); break;
        case 128: launch_umma<MB, NH, 2>(a, s); break;
        default: throw std::runtime_error("launch_latent_attention: unsupported row width");
    }
}

template <int MB>
void launch_umma_heads(const LatentAttnArgs& a, cudaStream_t s) {
    if (latent_tc_heads(a.heads) == 16) launch_umma_extra<MB, 16>(a, s);
    else launch_umma_extra<MB, 32>(a, s);
}

}  // namespace

LatentColumns latent_tc_columns(int kv_rank, int rot_width, int block_tokens) {
    LatentColumns c;
    if (block_tokens <= 0 || (block_tokens & (block_tokens - 1)) != 0) return c;
    c.values = (kv_rank + LU_COLS - 1) / LU_COLS * LU_COLS;
    c.rot0 = (kv_rank + 7) / 8 * 8;  // behind the vector, in its padding where there is room
    const int row = std::max(c.values, rot_width > 0 ? (c.rot0 + rot_width + 63) / 64 * 64 : 0);
    if (c.values <= 4 * LU_COLS && row <= c.values + 128) c.row = row;
    return c;
}

LatentColumns latent_general_columns(int kv_rank, int rot_width) {
    LatentColumns c;
    c.values = (kv_rank + 63) / 64 * 64;
    c.rot0 = (kv_rank + 7) / 8 * 8;
    c.row = std::max(c.values, rot_width > 0 ? (c.rot0 + rot_width + 63) / 64 * 64 : 0);
    return c;
}

int latent_tc_heads(int heads) { return heads <= 16 ? 16 : 32; }

int latent_max_shared_entries(int ctas) { return std::max(LA_SHARED_ROWS + LA_SHARED_ROWS / 2, LA_TARGET_CTAS / ctas) + 1; }
int latent_max_entries(int tokens, int ctas) { return std::max(tokens, latent_max_shared_entries(ctas)); }

void plan_latent_attention(const int32_t* start_pos, const int32_t* n_tokens, const int32_t* n_blocks, int lanes, int ctas, int wide_from,
                           bool shares, LatentPlan& plan, int window) {
    plan.entries.clear();
    plan.rows.clear();
    auto seen = [&](int pos) { return pos + 1 - attention_first_key(pos, window, 0); };  // keys of a position
    int rows = 0;
    int64_t keys = 0;
    for (int i = 0; i < lanes; ++i)
        if (n_tokens[i] < wide_from) {
            rows += n_tokens[i];
            for (int t = 0; t < n_tokens[i]; ++t) keys += seen(start_pos[i] + t);
        }
    // Every CTA should walk about the same number of keys and all of them fit on the GPU at once.  Once the rows alone fill it, only
    // a row more than twice as long as the mean is cut.
    int share = 1 << 30;
    if (shares && rows > 0 && rows <= LA_SHARED_ROWS) {
        const bool filled = rows * ctas >= LA_TARGET_CTAS;
        const int slots = filled ? rows + rows / 2 : std::max(rows, LA_TARGET_CTAS / ctas);
        share = (int)std::max<int64_t>(LA_MIN_SHARE, filled ? 2 * (keys / rows) : (keys + slots - 1) / slots);
        share = (share + LU_KEYS - 1) / LU_KEYS * LU_KEYS;
        for (;; share += LU_KEYS) {
            int64_t n = 0;
            for (int i = 0; i < lanes; ++i)
                if (n_tokens[i] < wide_from)
                    for (int t = 0; t < n_tokens[i]; ++t) n += std::min<int64_t>(LA_MAX_SHARES, (seen(start_pos[i] + t) - 1 + share) / share);
            if (n <= slots) break;
        }
    }
    int packed = 0, table_off = 0;
    for (int i = 0; i < lanes; packed += n_tokens[i], table_off += n_blocks[i], ++i) {
        if (n_tokens[i] >= wide_from) continue;
        for (int t = 0; t < n_tokens[i]; ++t) {
            const int pos = start_pos[i] + t, n = std::max(1, std::min(LA_MAX_SHARES, (int)(((int64_t)seen(pos) - 1 + share) / share)));
            const int first = plan.n_entries(), row = plan.n_rows();
            for (int k = 0; k < n; ++k)
                for (int32_t v : {row, k, n, pos, table_off, packed + t, first, 0}) plan.entries.push_back(v);
            plan.rows.push_back(packed + t);
        }
    }
}

void launch_latent_attention(const LatentAttnArgs& in, cudaStream_t s) {
    LatentAttnArgs a = in;
    if (a.n_entries <= 0) return;
    if (a.values == 0) a.values = a.rank;
    if (a.out.ld != a.values) throw std::runtime_error("launch_latent_attention: the output's rows are as wide as the latent");
    if (a.rot_dims > 0 && (a.rot0 % 8 != 0 || a.rot_dims % 2 != 0 || a.cos_t == nullptr || a.sin_t == nullptr))
        throw std::runtime_error("launch_latent_attention: a rotation starts at a multiple of 8 columns and needs its tables");
    if (a.q_h != nullptr) {
        if (!a.pool_f16 || a.out.h == nullptr) throw std::runtime_error("launch_latent_attention: f16 queries go with f16 pages and a bf16 output");
        if (a.status == nullptr) throw std::runtime_error("launch_latent_attention: the tensor-core kernel needs a status word");
        switch (a.values) {
            case 128: launch_umma_heads<1>(a, s); break;
            case 256: launch_umma_heads<2>(a, s); break;
            case 384: launch_umma_heads<3>(a, s); break;
            case 512: launch_umma_heads<4>(a, s); break;
            default: throw std::runtime_error("launch_latent_attention: unsupported rank");
        }
    } else {
        if (a.rank % 64 != 0 || a.values % 32 != 0 || a.rank > kLatentMaxRank) throw std::runtime_error("launch_latent_attention: latents above 1024 values are not supported");
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
