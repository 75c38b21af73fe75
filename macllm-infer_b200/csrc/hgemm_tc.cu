// Wide-batch matmul on the tcgen05 tensor cores over an f16 image of the weights.
//
// Replaces LinearOp::Quantized forward (src/model_weights.rs:346-377 of the reference) for prefill
// chunks: when hundreds of activation rows share one pass over a matrix, dequantising the GGUF blocks
// inside the GEMM repeats that work once per 128 tokens and the CUDA cores, not the tensor cores,
// set the pace.  A B200 has room to keep a second, f16 copy of every matrix (2 bytes per weight), made
// once at load time: w = f16(dequant(block)), one rounding per weight.  The GEMM is then the plain
// y[t][n] = sum_k xh[t][k] * wh[n][k] with f32 accumulation in tensor memory.
//
// One persistent CTA per SM, 320 threads in three roles:
//   warp 0   - one lane issues TMA loads (cp.async.bulk.tensor, 128-byte swizzle) of a 128 x 64 weight
//              box and a BN x 64 activation box per stage into a ring of shared-memory stages;
//   warp 1   - one lane issues the MMAs (tcgen05.mma kind::f16, M = 128 weight rows, N = BN tokens,
//              four K = 16 steps per stage), commits each stage back to the loader, and commits the tile
//              to the epilogue; two accumulators in tensor memory alternate so the next tile's main
//              loop runs under the previous tile's epilogue;
//   warps 2-9 - read the accumulator (tcgen05.ld, one lane per weight row, two warps per lane quadrant that take
//              every other 32 columns), apply scale / soft cap and store f32 results (32 consecutive rows of one
//              token per store instruction).  A tile's main loop is as long as K, its epilogue is not: with short K
//              it is the epilogue's instructions that count, hence eight warps and whole 32-column groups without
//              a test per column.
// Every mbarrier wait is bounded; a wait that gives up records a status word and the role leaves its
// loop, the other roles run into their own limits, and tensor memory is always released.
#include "hgemm_tc.h"
#include "kernels.h"
#include <cuda.h>
#include <cuda_bf16.h>
#include <mutex>

namespace mk {

namespace {

constexpr int HG_BM = 128;
constexpr int HG_BK = 64;  // 64 halves = 128 bytes = one swizzle row
constexpr int HG_EPI_THREADS = 256;
constexpr int HG_THREADS = 64 + HG_EPI_THREADS;
constexpr uint32_t HG_SPIN_LIMIT = 1u << 22;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void mbar_init(uint64_t* bar, uint32_t count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, uint32_t parity, uint32_t limit) {
    uint32_t addr = smem_u32(bar);
    for (uint32_t i = 0; i <= limit; ++i) {
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
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void mbar_expect_tx(uint64_t* bar, uint32_t bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes) : "memory");
}
// One 2-D box into this CTA's own shared memory; completes its bytes on the mbarrier.
__device__ __forceinline__ void tma_load_2d(void* dst, const void* tmap, int x, int y, uint64_t* bar) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
        ::"r"(smem_u32(dst)), "l"(tmap), "r"(x), "r"(y), "r"(smem_u32(bar))
        : "memory");
}
// K-major operand tile with 128-byte rows and the 128-byte swizzle: 8-row groups are 1024 bytes apart.
__device__ __forceinline__ uint64_t make_sw128_desc(uint32_t saddr) {
    uint64_t d = 0;
    d |= (uint64_t)((saddr >> 4) & 0x3FFF);
    d |= (uint64_t)1 << 16;                    // leading byte offset: unused for swizzled K-major tiles
    d |= (uint64_t)(1024 >> 4) << 32;          // stride byte offset
    d |= (uint64_t)1 << 46;                    // descriptor version for sm_100
    d |= (uint64_t)2 << 61;                    // layout type: 128-byte swizzle
    return d;
}
__device__ __forceinline__ void umma_f16(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}
__device__ __forceinline__ void umma_commit(uint64_t* bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t (&r)[32]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
        "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
          "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
          "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
          "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
        : "r"(taddr)
        : "memory");
}

// ---- load-time dequantisation to f16 (values as the reference's dequantize: crates candle k_quants
// to_float order of operations: (d * scale) * q - (dmin * min) in f32, then one rounding to f16) -------

__device__ __forceinline__ void q4k_scale_min(const uint8_t* sc, int j, int& s, int& m) {
    if (j < 4) {
        s = sc[j] & 63;
        m = sc[j + 4] & 63;
    } else {
        s = (sc[j + 4] & 0xF) | ((sc[j - 4] >> 6) << 4);
        m = (sc[j + 4] >> 4) | ((sc[j] >> 6) << 4);
    }
}

// One warp per 256-element block; lane l produces elements 8l .. 8l+7.  Row r of W goes to out + r * row_stride.
__global__ void dequant_f16_kernel(QWeight W, __half* out, int64_t row_stride) {
    const int64_t nb = W.cols / 256;
    const int64_t b = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (b >= W.rows * nb) return;
    const int lane = threadIdx.x & 31;
    __half h[8];
    if (W.type == QT_Q4_K) {
        const uint8_t* blk = (const uint8_t*)W.p0 + b * 144;
        float d = __half2float(*reinterpret_cast<const __half*>(blk));
        float dmin = __half2float(*reinterpret_cast<const __half*>(blk + 2));
        int j = lane >> 2;  // 32-element group
        int s, m;
        q4k_scale_min(blk + 4, j, s, m);
        float d1 = __fmul_rn(d, (float)s), m1 = __fmul_rn(dmin, (float)m);
        const uint8_t* qs = blk + 16 + (j >> 1) * 32 + (lane & 3) * 8;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            int q = (j & 1) ? (qs[i] >> 4) : (qs[i] & 0xF);
            h[i] = __float2half_rn(__fsub_rn(__fmul_rn(d1, (float)q), m1));
        }
    } else if (W.type == QT_Q6_K) {
        const uint8_t* ql = (const uint8_t*)W.p0 + b * 128;
        const uint8_t* qh = (const uint8_t*)W.p1 + b * 64;
        const int8_t* sc = (const int8_t*)W.p2 + b * 16;
        float d = __half2float(((const __half*)W.p3)[b]);
        int e0 = lane * 8;
        int hf = e0 >> 7, r = e0 & 127;     // 128-element half, offset inside it
        int grp = r >> 5, l0 = r & 31;       // which of the four 32-element quarters, first l
        float ds = __fmul_rn(d, (float)sc[hf * 8 + (l0 >> 4) + 2 * grp]);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            int l = l0 + i;
            uint8_t lo = ql[hf * 64 + (grp & 1) * 32 + l];
            int nib = (grp >> 1) ? (lo >> 4) : (lo & 0xF);
            int q = (nib | (((qh[hf * 32 + l] >> (2 * grp)) & 3) << 4)) - 32;
            h[i] = __float2half_rn(__fmul_rn(ds, (float)q));
        }
    } else if (W.type == QT_Q8_0) {
        int64_t row = b / nb, ib = b - row * nb;
        const int8_t* qs = (const int8_t*)W.p0 + row * W.cols + ib * 256 + lane * 8;
        float d = __half2float(((const __half*)W.p1)[row * (W.cols / 32) + ib * 8 + (lane >> 2)]);
#pragma unroll
        for (int i = 0; i < 8; ++i) h[i] = __float2half_rn(__fmul_rn(d, (float)qs[i]));
    } else {  // QT_F32
        const float* src = (const float*)W.p0 + b * 256 + lane * 8;
#pragma unroll
        for (int i = 0; i < 8; ++i) h[i] = __float2half_rn(src[i]);
    }
    const int64_t out_row = b / nb, out_blk = b - out_row * nb;
    *reinterpret_cast<uint4*>(out + out_row * row_stride + out_blk * 256 + lane * 8) = *reinterpret_cast<uint4*>(h);
}

// ---- the GEMM ------------------------------------------------------------------------------------

// Grouped form: one of the two matrices of a launch.
struct HgPart {
    int row_tiles, rows;      // row tiles of an expert's matrix, its true rows
    int T, k_blocks;          // rows (the second part), K blocks
    float* y;
    int ldy;
    __half* yh;
    int ldyh;
    float act_limit;          // of GatedAct::Clamped
    const float *act_pre, *act_post;
};

struct HgParams {
    int T, K, rows;
    float out_scale, softcap;
    int row_tiles, n_tiles;
    // split-K (narrow batches, long K): work item = (output tile, K share); every share writes its f32
    // partial sums to partial[share][T][rows] and the kernel that consumes the result adds the shares in
    // share order, so the value does not depend on scheduling and no extra pass over the output is needed
    int splits, kb_per_split;
    float* partial;
    int32_t* status;
    // gated epilogue (splits == 1): weight rows 2j / 2j+1 are the gate / up projections of feature j and the kernel
    // writes yh[t][j] = f16(act(gate, up)) instead of y; 0 = off, otherwise 1 + GatedAct::Kind
    int gated;
    int bf16;  // both operands (and yh) are bfloat16
    // stacked projections with inputs of their own: the first row of input g in the activation matrix is g * T
    int n_groups;
    int group_end[kMaxRowGroups];
    int group_tiles;
    int scattered;  // the result goes where `scatter` says (splits == 1)
    MatmulScatter scatter;
    // activation rows grouped by expert, beside them a matrix that rows of its own meet all of (see HgPart); item = (part, expert,
    // row tile, token tile of the expert's rows)
    int experts;
    int box_rows;             // rows of an activation box
    const int32_t* offsets;   // [experts + 1]
    HgPart part[2];
};
constexpr int HG_MAX_EXPERTS = 1024;

// One output tile: the first weight row, the first activation row, and the bounds of what counts.
struct HgTile {
    int w_row, row0;          // weight row of the tile (within the whole image), output row it becomes
    int x_row, tok0, tok_end; // activation row of the tile (box), its first output row, end of the output rows
    int rows;                 // end of the output columns
    int part;                 // grouped: 0 experts, 1 the matrix beside them
};

// Rows shared out evenly over as few tiles of at most `most` rows as hold them, in steps of 16.
__device__ __forceinline__ int even_tile(int n, int most) {
    const int tiles = (n + most - 1) / most;
    return ((n + tiles - 1) / tiles + 15) & ~15;
}

__device__ __forceinline__ int group_row0(const HgParams& p, int m_tile) {
    if (p.n_groups == 1) return 0;
    if (p.group_tiles > 0) return m_tile / p.group_tiles * p.T;
    int g = 0;
    while (g < p.n_groups - 1 && m_tile >= p.group_end[g]) ++g;
    return g * p.T;
}

template <int BN, int STAGES>
struct HgSmem {
    static constexpr int A_BYTES = HG_BM * HG_BK * 2;   // 16 KiB
    static constexpr int B_BYTES = BN * HG_BK * 2;
    static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
    static constexpr size_t TOTAL = (size_t)STAGES * STAGE_BYTES + 1024 /* alignment slack */ + 256 /* barriers */;
};

__device__ __forceinline__ float finish_value(float v, const HgParams& p) {
    v *= p.out_scale;
    if (p.softcap != 0.f) v = tanhf(v * (1.0f / p.softcap)) * p.softcap;
    return v;
}

// The activations of the gated feed-forward, as the SwiGLU kernel of quantize.cu computes them.
__device__ __forceinline__ float hg_sigmoid(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }  // to what a 16-bit result needs
__device__ __forceinline__ float hg_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float hg_clamped(float g, float u, float limit) {  // clamped_gate_f to what the 16-bit result needs
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return __fdividef(g, 1.0f + __expf(-1.702f * g)) * (u + 1.0f);
}
__device__ __forceinline__ float hg_gelu_tanh(float x) {
    return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * x * (1.0f + 0.044715f * x * x)));
}

// GATED: scattered results are multiplied by a gate (MatmulScatter::gate).
template <int BN, int STAGES, bool GATED>
__global__ void __launch_bounds__(HG_THREADS, 1)
hgemm_tc_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, const __grid_constant__ CUtensorMap tm_w1,
                const __grid_constant__ CUtensorMap tm_x1, const __grid_constant__ HgParams p) {
    using L = HgSmem<BN, STAGES>;
    constexpr int LD_COLS = BN >= 32 ? 32 : BN;
    extern __shared__ uint8_t hg_smem_raw[];
    __shared__ int32_t first_item[HG_MAX_EXPERTS + 1];  // grouped by expert: items of the experts before
    __shared__ int32_t first_row[HG_MAX_EXPERTS + 1];
    uint8_t* tiles = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(hg_smem_raw) + 1023) & ~(uintptr_t)1023);
    uint64_t* bars = reinterpret_cast<uint64_t*>(tiles + (size_t)STAGES * L::STAGE_BYTES);
    uint64_t* full = bars;                  // [STAGES]  loader -> MMA
    uint64_t* empty = bars + STAGES;        // [STAGES]  MMA -> loader
    uint64_t* acc_full = bars + 2 * STAGES; // [2]       MMA -> epilogue
    uint64_t* acc_empty = acc_full + 2;     // [2]       epilogue -> MMA
    __shared__ uint32_t tmem_base_slot;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int k_blocks = p.K / HG_BK;
    const int mn_tiles = p.row_tiles * p.n_tiles;
    int total_items = mn_tiles * p.splits;
    constexpr uint32_t TMEM_COLS = 2 * BN < 32 ? 32 : 2 * BN;

    if (threadIdx.x == 0) {
        for (int i = 0; i < STAGES; ++i) {
            mbar_init(&full[i], 1);
            mbar_init(&empty[i], 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(&acc_full[i], 1);
            mbar_init(&acc_empty[i], HG_EPI_THREADS);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_slot)),
                     "r"(TMEM_COLS)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem_base = tmem_base_slot;
    // Everything above is private to the CTA.  The weights do not depend on the predecessor kernel either, so
    // the loader fills the ring with weight boxes first and only then waits for the predecessor, whose output
    // (the activations) it loads next.  Every other access to global memory of this kernel (the epilogue's
    // stores) is ordered after those loads through the mbarriers.
    pdl_trigger();
    if (p.experts > 0) {
        // the row ranges are the predecessor's: one warp turns them into item numbers
        pdl_wait();
        if (warp == 0) {
            const HgPart& every = p.part[1];
            int carry = every.T > 0 ? (every.T + BN - 1) / BN * every.row_tiles : 0;
            for (int base = 0; base < p.experts; base += 32) {
                const int e = base + lane;
                int lo = 0, n = 0;
                if (e < p.experts) {
                    lo = p.offsets[e];
                    n = (p.offsets[e + 1] - lo + BN - 1) / BN * p.part[0].row_tiles;
                }
                int inc = n;
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const int v = __shfl_up_sync(0xffffffffu, inc, o);
                    if (lane >= o) inc += v;
                }
                if (e < p.experts) {
                    first_item[e] = carry + inc - n;
                    first_row[e] = lo;
                }
                carry += __shfl_sync(0xffffffffu, inc, 31);
            }
            if (lane == 0) {
                first_item[p.experts] = carry;
                first_row[p.experts] = p.offsets[p.experts];
            }
        }
        __syncthreads();
        total_items = first_item[p.experts];
    }

    // work item -> (row tile, token tile, K share); token tiles vary fastest, so the CTAs that run side by side cover
    // a few row tiles across every token tile: each weight box comes from HBM once and the activations stay in L2
    auto decode = [&](int item, HgTile& t, int& kb0, int& kb1) {
        if (p.experts > 0) {
            int e = 0, first = 0, row = 0, n = p.part[1].T;
            t.part = item < first_item[0] ? 1 : 0;
            if (t.part == 0) {
                // the last expert whose items begin at or before this one; experts without rows have none
                for (int step = HG_MAX_EXPERTS; step > 0; step >>= 1)
                    if (e + step < p.experts && first_item[e + step] <= item) e += step;
                first = first_item[e];
                row = first_row[e];
                n = first_row[e + 1] - row;
            }
            const HgPart& part = p.part[t.part];
            const int mn = item - first, n_tiles = (n + BN - 1) / BN, m_tile = mn / n_tiles, each = even_tile(n, BN);
            t.w_row = (e * part.row_tiles + m_tile) * HG_BM;
            t.row0 = m_tile * HG_BM;
            t.x_row = t.tok0 = row + mn % n_tiles * each;
            t.tok_end = min(row + n, t.tok0 + each);
            t.rows = part.rows;
            kb0 = 0;
            kb1 = part.k_blocks;
            return;
        }
        t.part = 0;
        const int mn = item % mn_tiles, split = item / mn_tiles, m_tile = mn / p.n_tiles;
        t.w_row = t.row0 = m_tile * HG_BM;
        t.tok0 = mn % p.n_tiles * BN;
        t.x_row = group_row0(p, m_tile) + t.tok0;
        t.tok_end = p.T;
        t.rows = p.rows;
        kb0 = split * p.kb_per_split;
        kb1 = min(k_blocks, kb0 + p.kb_per_split);
    };

    if (warp == 0) {
        // ---- loader
        if (lane == 0) {
            uint32_t it = 0;
            bool ok = true, waited = p.experts > 0;
            int held_x[STAGES], held_y[STAGES];  // activation boxes of the stages filled before the wait
            for (int item = blockIdx.x; item < total_items && ok; item += gridDim.x) {
                HgTile tile;
                int kb0, kb1;
                decode(item, tile, kb0, kb1);
                for (int kb = kb0; kb < kb1; ++kb, ++it) {
                    const uint32_t st = it % STAGES, ph = (it / STAGES) & 1;
                    if (it == STAGES && !waited) {  // the ring is full of weights: now the activations
                        pdl_wait();
                        waited = true;
                        for (int h = 0; h < STAGES; ++h)
                            tma_load_2d(tiles + (size_t)h * L::STAGE_BYTES + L::A_BYTES, &tm_x, held_x[h], held_y[h], &full[h]);
                    }
                    if (!mbar_wait(&empty[st], ph ^ 1, HG_SPIN_LIMIT)) {
                        atomicExch(p.status, 11);
                        ok = false;
                        break;
                    }
                    uint8_t* a_dst = tiles + (size_t)st * L::STAGE_BYTES;
                    uint8_t* b_dst = a_dst + L::A_BYTES;
                    if (p.experts > 0) {
                        // as many activation boxes as the tile has rows for
                        const int boxes = (max(tile.tok_end - tile.tok0, 1) + p.box_rows - 1) / p.box_rows;
                        mbar_expect_tx(&full[st], (uint32_t)(L::A_BYTES + boxes * p.box_rows * HG_BK * 2));
                        tma_load_2d(a_dst, tile.part == 0 ? &tm_w : &tm_w1, kb * HG_BK, tile.w_row, &full[st]);
                        for (int b = 0; b < boxes; ++b)
                            tma_load_2d(b_dst + b * p.box_rows * HG_BK * 2, tile.part == 0 ? &tm_x : &tm_x1, kb * HG_BK, tile.x_row + b * p.box_rows, &full[st]);
                        continue;
                    }
                    mbar_expect_tx(&full[st], (uint32_t)L::STAGE_BYTES);
                    tma_load_2d(a_dst, &tm_w, kb * HG_BK, tile.w_row, &full[st]);
                    if (waited) {
                        tma_load_2d(b_dst, &tm_x, kb * HG_BK, tile.x_row, &full[st]);
                    } else {
                        held_x[st] = kb * HG_BK;
                        held_y[st] = tile.x_row;
                    }
                }
            }
            if (!waited) {  // fewer stages of work than the ring holds
                pdl_wait();
                for (uint32_t h = 0; h < it && h < (uint32_t)STAGES; ++h)
                    tma_load_2d(tiles + (size_t)h * L::STAGE_BYTES + L::A_BYTES, &tm_x, held_x[h], held_y[h], &full[h]);
            }
        }
    } else if (warp == 1) {
        // ---- MMA issuer
        if (lane == 0) {
            const uint32_t idesc_wide = (1u << 4) | (p.bf16 ? (1u << 7) | (1u << 10) : 0u) | ((uint32_t)(HG_BM >> 4) << 24);
            uint32_t it = 0, tile_it = 0;
            bool ok = true;
            for (int item = blockIdx.x; item < total_items && ok; item += gridDim.x, ++tile_it) {
                HgTile tile;
                int kb0, kb1;
                decode(item, tile, kb0, kb1);
                const uint32_t acc = tile_it & 1, acc_ph = (tile_it >> 1) & 1;
                if (!mbar_wait(&acc_empty[acc], acc_ph ^ 1, HG_SPIN_LIMIT)) {
                    atomicExch(p.status, 12);
                    break;
                }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t d_tmem = tmem_base + acc * BN;
                // grouped: no wider than the tile's rows, in steps of 16
                const uint32_t wide = p.experts > 0 ? (uint32_t)((tile.tok_end - tile.tok0 + 15) & ~15) : (uint32_t)BN;
                const uint32_t idesc = idesc_wide | ((wide >> 3) << 17);
                for (int kb = kb0; kb < kb1; ++kb, ++it) {
                    const uint32_t st = it % STAGES, ph = (it / STAGES) & 1;
                    if (!mbar_wait(&full[st], ph, HG_SPIN_LIMIT)) {
                        atomicExch(p.status, 13);
                        ok = false;
                        break;
                    }
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint32_t a_addr = smem_u32(tiles + (size_t)st * L::STAGE_BYTES);
                    const uint32_t b_addr = a_addr + L::A_BYTES;
                    const uint64_t adesc = make_sw128_desc(a_addr), bdesc = make_sw128_desc(b_addr);
#pragma unroll
                    for (int k = 0; k < HG_BK / 16; ++k) {
                        // 16 halves = 32 bytes further along K inside the swizzled row: +2 in 16-byte units
                        umma_f16(d_tmem, adesc + (uint64_t)(2 * k), bdesc + (uint64_t)(2 * k), idesc, (kb > kb0 || k > 0) ? 1u : 0u);
                    }
                    umma_commit(&empty[st]);
                }
                if (ok) umma_commit(&acc_full[acc]);
            }
        }
    } else {
        // ---- epilogue: warps 2..9 own TMEM lane quadrants (warp % 4), two each
        const int quad = warp & 3, odd_group = (warp - 2) >> 2;
        const int etid = (int)threadIdx.x - 64;  // among the epilogue threads
        const bool plain = p.out_scale == 1.0f && p.softcap == 0.f;
        if (GATED || p.part[0].act_post != nullptr) pdl_wait();   // the factors of the rows, or the gates, come from a predecessor
        uint32_t tile_it = 0;
        for (int item = blockIdx.x; item < total_items; item += gridDim.x, ++tile_it) {
            HgTile tile;
            int kb0, kb1;
            decode(item, tile, kb0, kb1);
            const int split = p.splits > 1 ? item / mn_tiles : 0;
            const uint32_t acc = tile_it & 1, acc_ph = (tile_it >> 1) & 1;
            // every epilogue warp waits for itself, then all agree on the outcome, so that a wait that
            // gave up takes all of them out of the loop together (they meet again at named barrier 1)
            const uint32_t got = mbar_wait(&acc_full[acc], acc_ph, HG_SPIN_LIMIT) ? 1u : 0u;
            uint32_t all_got;
            asm volatile(
                "{\n\t.reg .pred p, q;\n\t"
                "setp.ne.u32 q, %1, 0;\n\t"
                "bar.red.and.pred p, 1, %2, q;\n\t"
                "selp.u32 %0, 1, 0, p;\n\t}"
                : "=r"(all_got)
                : "r"(got), "n"(HG_EPI_THREADS)
                : "memory");
            if (!all_got) {
                if (etid == 0) atomicExch(p.status, 14);
                break;
            }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int row = tile.row0 + quad * 32 + lane;
            const int tok0 = tile.tok0;
            const HgPart& part = p.part[tile.part];  // where a whole tile goes and its activation's constants (both forms)
            float* dst = p.splits > 1 ? p.partial + (int64_t)split * p.T * p.rows : part.y;
            const int ld = p.splits > 1 ? p.rows : part.ldy;
#pragma unroll 1
            for (int cb = odd_group * LD_COLS; cb < BN; cb += 2 * LD_COLS) {
                if (tok0 + cb >= tile.tok_end) break;  // uniform over the warp: nothing but padding from here on
                // the factors of the chunk's tokens, one per lane, on their way with the accumulators
                float pre = 1.0f, post = 1.0f;
                if (p.gated == 1 + GatedAct::Clamped && tok0 + cb + lane < tile.tok_end) {
                    if (part.act_pre != nullptr) pre = part.act_pre[tok0 + cb + lane];
                    if (part.act_post != nullptr) post = part.act_post[tok0 + cb + lane];
                }
                uint32_t r[32];
                tmem_ld32(tmem_base + ((uint32_t)(quad * 32) << 16) + acc * BN + (uint32_t)cb, r);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (p.gated != 0) {
                    // lanes 2i / 2i+1 hold gate / up of one feature: the even lane finishes the even token columns,
                    // the odd lane the odd ones, after one exchange per pair of columns
                    const bool odd = (lane & 1) != 0;
                    const int feature = row >> 1;
                    const bool weighed = part.act_pre != nullptr || part.act_post != nullptr;
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        float mine = __uint_as_float(odd ? r[i] : r[i + 1]);       // what the partner needs
                        float theirs = __shfl_xor_sync(0xffffffffu, mine, 1);
                        float g = odd ? theirs : __uint_as_float(r[i]);
                        float u = odd ? __uint_as_float(r[i + 1]) : theirs;
                        int tok = tok0 + cb + i + (odd ? 1 : 0);
                        float w_in = 1.0f, w_out = 1.0f;
                        if (weighed) {  // uniform
                            w_in = __shfl_sync(0xffffffffu, pre, i + (odd ? 1 : 0));
                            w_out = __shfl_sync(0xffffffffu, post, i + (odd ? 1 : 0));
                        }
                        if (row < tile.rows && tok < tile.tok_end) {
                            float a;
                            if (p.gated == 1 + GatedAct::Clamped) {
                                a = hg_clamped(w_in * g, w_in * u, part.act_limit) * w_out;
                            } else {
                                a = (p.gated == 1 + GatedAct::Silu ? hg_silu(g) : hg_gelu_tanh(g)) * u;
                            }
                            if (p.bf16) reinterpret_cast<__nv_bfloat16*>(part.yh)[(int64_t)tok * part.ldyh + feature] = __float2bfloat16_rn(a);
                            else part.yh[(int64_t)tok * part.ldyh + feature] = __float2half_rn(a);
                        }
                    }
                } else if (p.scattered != 0 && p.scatter.rest != nullptr && row >= p.scatter.rest_from) {
                    float* out = p.scatter.rest + (int64_t)(tok0 + cb) * p.scatter.ld_rest + row - p.scatter.rest_from;
                    if (row < tile.rows) {
#pragma unroll
                        for (int i = 0; i < 32; ++i, out += p.scatter.ld_rest)
                            if (tok0 + cb + i < tile.tok_end) *out = __uint_as_float(r[i]);
                    }
                } else if (p.scattered != 0 && p.scatter.type == MatmulScatter::BF16 && p.scatter.row_map == nullptr && p.scatter.block_shift == 31 && !GATED) {
                    const int64_t col = row < tile.rows ? p.scatter.column(row) : -1;
                    if (col >= 0) {
                        __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.scatter.out) + (int64_t)(tok0 + cb) * p.scatter.ld_row + col;
#pragma unroll
                        for (int i = 0; i < 32; ++i, out += p.scatter.ld_row)
                            if (tok0 + cb + i < tile.tok_end) *out = __float2bfloat16_rn(__uint_as_float(r[i]));
                    }
                } else if (GATED && p.scattered != 0) {
                    const int64_t col = row < tile.rows ? p.scatter.column(row) : -1;
                    if (col >= 0) {
#pragma unroll 1
                        for (int i0 = 0; i0 < 32; i0 += 8) {  // the gates of eight tokens on their way together
                            float z[8];
#pragma unroll
                            for (int i = 0; i < 8; ++i) z[i] = tok0 + cb + i0 + i < tile.tok_end ? p.scatter.gate_sum(tok0 + cb + i0 + i, row) : 0.f;
#pragma unroll
                            for (int i = 0; i < 8; ++i) {
                                const int tok = tok0 + cb + i0 + i;
                                const float v = __uint_as_float(i0 == 0 ? r[i] : (i0 == 8 ? r[8 + i] : (i0 == 16 ? r[16 + i] : r[24 + i])));
                                if (tok < tile.tok_end) p.scatter.put(p.scatter.row(tok) + col, v * hg_sigmoid(z[i]));
                            }
                        }
                    }
                } else if (p.scattered != 0) {
                    const int64_t col = row < tile.rows ? p.scatter.column(row) : -1;
                    if (col >= 0) {
#pragma unroll
                        for (int i = 0; i < 32; ++i) {
                            const int tok = tok0 + cb + i;
                            if (tok < tile.tok_end) p.scatter.put(p.scatter.row(tok) + col, __uint_as_float(r[i]));
                        }
                    }
                } else if (row < tile.rows && plain && tok0 + cb + 32 <= tile.tok_end) {
                    float* out = dst + (int64_t)(tok0 + cb) * ld + row;
#pragma unroll
                    for (int i = 0; i < 32; ++i, out += ld) *out = __uint_as_float(r[i]);
                } else if (row < tile.rows) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        int tok = tok0 + cb + i;
                        if (tok < tile.tok_end) {
                            float v = __uint_as_float(r[i]);
                            if (p.splits == 1) v = finish_value(v, p);
                            dst[(int64_t)tok * ld + row] = v;
                        }
                    }
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(&acc_empty[acc]);
        }
    }

    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(TMEM_COLS) : "memory");
    }
}

// ---- host side --------------------------------------------------------------------------------------

using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiledFn encode_fn() {
    static EncodeTiledFn fn = nullptr;
    static std::once_flag once;
    std::call_once(once, [] {
        void* sym = nullptr;
        cudaDriverEntryPointQueryResult q = cudaDriverEntryPointSymbolNotFound;
        cudaError_t e = cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &q);
        if (e == cudaSuccess && q == cudaDriverEntryPointSuccess) fn = reinterpret_cast<EncodeTiledFn>(sym);
    });
    if (fn == nullptr) throw std::runtime_error("the CUDA driver does not provide cuTensorMapEncodeTiled");
    return fn;
}

// 16-bit matrix [n_rows][cols] row-major, boxes of box_rows x 64 columns, 128-byte swizzle, zero fill.
void encode_half_matrix(CUtensorMap* out, const void* base, int64_t n_rows, int64_t cols, int box_rows, bool bf16 = false) {
    if ((reinterpret_cast<uintptr_t>(base) & 15) != 0) throw std::runtime_error("hgemm: matrix base must be 16-byte aligned");
    cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)n_rows};
    cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
    cuuint32_t box[2] = {(cuuint32_t)HG_BK, (cuuint32_t)box_rows};
    cuuint32_t elem[2] = {1, 1};
    CUresult r = encode_fn()(out, bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 2, const_cast<void*>(base), dims, strides,
                             box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) throw std::runtime_error("cuTensorMapEncodeTiled failed with code " + std::to_string((int)r));
}

template <int BN, int STAGES>
void launch_hg(const CUtensorMap& tw, const CUtensorMap& tx, const CUtensorMap& tw1, const CUtensorMap& tx1, const HgParams& p, int grid, cudaStream_t s) {
    constexpr size_t smem = HgSmem<BN, STAGES>::TOTAL;
    auto* kernel = p.scattered != 0 && p.scatter.gate != nullptr ? hgemm_tc_kernel<BN, STAGES, true> : hgemm_tc_kernel<BN, STAGES, false>;
    ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), smem);
    launch_pdl(kernel, dim3(grid), dim3(HG_THREADS), smem, s, tw, tx, tw1, tx1, p);
    MK_LAUNCH_CHECK();
}

void launch_hg_width(int bn, const CUtensorMap& tw, const CUtensorMap& tx, const CUtensorMap& tw1, const CUtensorMap& tx1, const HgParams& p, int grid, cudaStream_t s) {
    if (bn == 256) launch_hg<256, 4>(tw, tx, tw1, tx1, p, grid, s);
    else if (bn == 128) launch_hg<128, 6>(tw, tx, tw1, tx1, p, grid, s);
    else launch_hg<64, 8>(tw, tx, tw1, tx1, p, grid, s);
}

}  // namespace

void encode_tma_2d(void* out_map, bool bytes_not_halves, const void* base, uint64_t inner, uint64_t outer, uint64_t row_stride_bytes,
                   uint32_t box_inner, uint32_t box_outer, bool swizzle_128b) {
    if ((reinterpret_cast<uintptr_t>(base) & 15) != 0 || row_stride_bytes % 16 != 0)
        throw std::runtime_error("TMA descriptor: base and row stride must be multiples of 16 bytes");
    cuuint64_t dims[2] = {(cuuint64_t)inner, (cuuint64_t)outer};
    cuuint64_t strides[1] = {(cuuint64_t)row_stride_bytes};
    cuuint32_t box[2] = {(cuuint32_t)box_inner, (cuuint32_t)box_outer};
    cuuint32_t elem[2] = {1, 1};
    CUresult r = encode_fn()(reinterpret_cast<CUtensorMap*>(out_map),
                             bytes_not_halves ? CU_TENSOR_MAP_DATA_TYPE_UINT8 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 2,
                             const_cast<void*>(base), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                             swizzle_128b ? CU_TENSOR_MAP_SWIZZLE_128B : CU_TENSOR_MAP_SWIZZLE_NONE,
                             CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) throw std::runtime_error("cuTensorMapEncodeTiled failed with code " + std::to_string((int)r));
}



bool hgemm_tc_supported(const QWeight& W) {
    if (W.type != QT_Q4_K && W.type != QT_Q6_K && W.type != QT_Q8_0 && W.type != QT_F32) return false;
    return W.cols % 256 == 0 && W.rows > 0;
}

void build_half_weight_stacked(const QWeight* const* parts, int n_parts, HalfWeight& out, cudaStream_t s) {
    if (n_parts <= 0) throw std::runtime_error("build_half_weight: nothing to build");
    int64_t rows = 0;
    const int64_t cols = parts[0]->cols;
    for (int i = 0; i < n_parts; ++i) {
        if (!hgemm_tc_supported(*parts[i]) || parts[i]->cols != cols) throw std::runtime_error("build_half_weight: unsupported matrix");
        rows += parts[i]->rows;
    }
    out.rows = rows;
    out.cols = cols;
    out.values.alloc((size_t)rows * (size_t)cols * 2);
    int64_t row0 = 0;
    for (int i = 0; i < n_parts; ++i) {
        const QWeight& W = *parts[i];
        const int64_t blocks = W.rows * (W.cols / 256);
        const int warps_per_cta = 8;
        dequant_f16_kernel<<<(unsigned)((blocks + warps_per_cta - 1) / warps_per_cta), warps_per_cta * 32, 0, s>>>(
            W, out.values.as<__half>() + row0 * cols, cols);
        MK_LAUNCH_CHECK();
        row0 += W.rows;
    }
    static_assert(sizeof(CUtensorMap) <= sizeof(out.tmap), "descriptor storage too small");
    encode_half_matrix(reinterpret_cast<CUtensorMap*>(out.tmap), out.values.ptr(), rows, cols, HG_BM);
    out.ready = true;
}

void build_half_weight_interleaved(const QWeight& gate, const QWeight& up, HalfWeight& out, cudaStream_t s) {
    if (!hgemm_tc_supported(gate) || !hgemm_tc_supported(up) || gate.cols != up.cols || gate.rows != up.rows)
        throw std::runtime_error("build_half_weight_interleaved: unsupported pair of matrices");
    const int64_t cols = gate.cols;
    out.rows = 2 * gate.rows;
    out.cols = cols;
    out.values.alloc((size_t)out.rows * (size_t)cols * 2);
    const QWeight* parts[2] = {&gate, &up};
    for (int i = 0; i < 2; ++i) {
        const int64_t blocks = parts[i]->rows * (cols / 256);
        const int warps_per_cta = 8;
        dequant_f16_kernel<<<(unsigned)((blocks + warps_per_cta - 1) / warps_per_cta), warps_per_cta * 32, 0, s>>>(
            *parts[i], out.values.as<__half>() + i * cols, 2 * cols);
        MK_LAUNCH_CHECK();
    }
    encode_half_matrix(reinterpret_cast<CUtensorMap*>(out.tmap), out.values.ptr(), out.rows, cols, HG_BM);
    out.ready = true;
}

void build_bf16_weight(const float* values, int64_t rows, int64_t cols, HalfWeight& out, cudaStream_t s, const std::vector<int64_t>& group_rows) {
    if (rows <= 0 || cols <= 0 || cols % HG_BK != 0) throw std::runtime_error("build_bf16_weight: columns must be padded to a multiple of 64");
    if (group_rows.size() > (size_t)kMaxRowGroups) throw std::runtime_error("build_bf16_weight: too many stacked projections");
    std::vector<__nv_bfloat16> bits((size_t)(rows * cols));
#pragma omp parallel for
    for (int64_t i = 0; i < rows * cols; ++i) bits[(size_t)i] = __float2bfloat16_rn(values[i]);
    out.rows = rows;
    out.cols = cols;
    out.bf16 = true;
    out.n_groups = 1;
    if (group_rows.size() > 1) {
        out.n_groups = (int)group_rows.size();
        int64_t end = 0;
        for (size_t g = 0; g < group_rows.size(); ++g) {
            if (group_rows[g] % HG_BM != 0) throw std::runtime_error("build_bf16_weight: a stacked projection must be a multiple of 128 rows");
            end += group_rows[g];
            out.group_end[g] = (int)(end / HG_BM);
        }
        if (end != rows) throw std::runtime_error("build_bf16_weight: stacked projections do not add up");
    }
    out.values.upload(bits.data(), bits.size() * 2, s);
    MK_CUDA(cudaStreamSynchronize(s));
    encode_half_matrix(reinterpret_cast<CUtensorMap*>(out.tmap), out.values.ptr(), rows, cols, HG_BM, true);
    out.ready = true;
}

void build_bf16_weight_groups(const float* values, int64_t rows, int64_t cols, int groups, HalfWeight& out, cudaStream_t s) {
    if (groups <= 0 || rows % groups != 0 || rows / groups % HG_BM != 0)
        throw std::runtime_error("build_bf16_weight_groups: every stacked projection must be a multiple of 128 rows");
    build_bf16_weight(values, rows, cols, out, s);
    out.n_groups = groups;
    out.group_tiles = (int)(rows / groups / HG_BM);
}

void build_half_weight(const QWeight& W, HalfWeight& out, cudaStream_t s) {
    const QWeight* one = &W;
    build_half_weight_stacked(&one, 1, out, s);
}

HgemmPlan hgemm_tc_plan(int64_t rows, int64_t cols, int T, int max_splits) {
    HgemmPlan pl;
    pl.bn = T <= 64 ? 64 : 128;
    if (T > 128) {
        // 256-token tiles do about 10 % more per unit of time (less shared-memory traffic per MMA, half the epilogue
        // hand-offs), 128-token tiles fill the last round of CTAs better: take the one with fewer (rounds x tile time)
        const int64_t mt = (rows + HG_BM - 1) / HG_BM;
        const double cost256 = (double)((mt * ((T + 255) / 256) + 147) / 148) * 2.0;
        const double cost128 = (double)((mt * ((T + 127) / 128) + 147) / 148) * 1.1;
        pl.bn = cost128 < cost256 ? 128 : 256;
    }
    pl.row_tiles = (int)((rows + HG_BM - 1) / HG_BM);
    pl.n_tiles = (T + pl.bn - 1) / pl.bn;
    const int kb = (int)(cols / HG_BK);
    const int tiles = pl.row_tiles * pl.n_tiles;
    const int sms = 148;
    // shares of K per output tile: fewest "waves x (K blocks per share + fixed cost)" with shares of at least
    // four K blocks and at most 16 MiB of partial sums
    int best = 1;
    long best_cost = -1;
    for (int s = 1; s <= std::max(1, std::min(max_splits, 16)); ++s) {
        int per = (kb + s - 1) / s;
        if (s > 1 && (per < 4 || (size_t)s * T * rows * 4 > ((size_t)16 << 20))) break;
        if ((kb + per - 1) / per != s) continue;  // not a distinct split
        long waves = ((long)tiles * s + sms - 1) / sms;
        long cost = waves * (per + 3) + (s > 1 ? 1 : 0);
        if (best_cost < 0 || cost < best_cost) { best_cost = cost; best = s; }
    }
    pl.splits = best;
    pl.kb_per_split = (kb + best - 1) / best;
    pl.partial_floats = best > 1 ? (size_t)best * T * rows : 0;
    return pl;
}

namespace {
int launch_hgemm_any(const HalfWeight& W, const __half* xh, int T, float* y, int ldy, float out_scale, float softcap,
                     const HgemmScratch& ws, cudaStream_t s, int max_splits, const GatedAct* act, __half* yh, int ldyh,
                     const MatmulScatter* scatter = nullptr);
}

int launch_hgemm_tc(const HalfWeight& W, const __half* xh, int T, float* y, int ldy, float out_scale, float softcap,
                    const HgemmScratch& ws, cudaStream_t s, int max_splits) {
    return launch_hgemm_any(W, xh, T, y, ldy, out_scale, softcap, ws, s, max_splits, nullptr, nullptr, 0);
}

void launch_hgemm_tc_scatter(const HalfWeight& W, const __half* xh, int T, const MatmulScatter& to, const HgemmScratch& ws, cudaStream_t s) {
    if (to.out == nullptr || to.part_rows <= 0) throw std::runtime_error("launch_hgemm_tc_scatter: no destination");
    launch_hgemm_any(W, xh, T, nullptr, 0, 1.0f, 0.f, ws, s, 1, nullptr, nullptr, 0, &to);
}

void launch_hgemm_tc_gated(const HalfWeight& W, const __half* xh, int T, const GatedAct& act, __half* yh, int ldyh, const HgemmScratch& ws,
                           cudaStream_t s) {
    if (W.rows % 2 != 0 || yh == nullptr) throw std::runtime_error("launch_hgemm_tc_gated: needs an interleaved gate/up image and an output");
    launch_hgemm_any(W, xh, T, nullptr, 0, 1.0f, 0.f, ws, s, 1, &act, yh, ldyh);
}

void launch_hgemm_tc_experts(const ExpertRows& experts, const ExpertRows* every, const HgemmScratch& ws, cudaStream_t s) {
    if (experts.experts <= 0 || experts.experts > HG_MAX_EXPERTS || experts.offsets == nullptr) throw std::runtime_error("launch_hgemm_tc_experts: 1 to 1024 experts");
    if (experts.T <= 0) return;
    HgParams p{};
    CUtensorMap tx[2];
    const CUtensorMap* tw[2] = {};
    int most_items = 0;
    // token tiles about as wide as an expert has rows
    const int mean = (experts.T + experts.experts - 1) / experts.experts;
    const int bn = mean <= 48 ? 64 : (mean <= 160 ? 128 : 256);
    p.box_rows = bn == 64 ? 16 : 64;
    for (int i = 0; i < 2; ++i) {
        const ExpertRows* e = i == 0 ? &experts : every;
        if (e == nullptr) {
            tw[1] = tw[0];
            tx[1] = tx[0];
            continue;
        }
        const HalfWeight& W = *e->W;
        if (!W.ready || e->xh == nullptr || e->rows_padded % HG_BM != 0 || W.rows != (int64_t)e->experts * e->rows_padded || W.n_groups != 1)
            throw std::runtime_error("launch_hgemm_tc_experts: matrices of whole 128-row tiles and their rows");
        if ((e->act != nullptr) != (e->yh != nullptr) || (experts.act != nullptr) != (e->act != nullptr) || W.bf16 != experts.W->bf16 || (i == 1 && e->experts != 1))
            throw std::runtime_error("launch_hgemm_tc_experts: the two parts differ in form");
        tw[i] = reinterpret_cast<const CUtensorMap*>(W.tmap);
        encode_half_matrix(&tx[i], e->xh, e->T, W.cols, p.box_rows, W.bf16);
        HgPart& part = p.part[i];
        part.row_tiles = e->rows_padded / HG_BM;
        part.rows = e->rows;
        part.T = i == 1 ? e->T : 0;
        part.k_blocks = (int)(W.cols / HG_BK);
        part.y = e->y;
        part.ldy = e->ldy;
        part.yh = e->yh;
        part.ldyh = e->ldyh;
        if (e->act != nullptr) {
            part.act_limit = e->act->limit;
            part.act_pre = e->act->pre;
            part.act_post = e->act->post;
        }
        most_items += part.row_tiles * (std::min(e->T, e->experts) + e->T / bn);
    }
    p.T = experts.T;
    p.K = (int)experts.W->cols;
    p.rows = (int)experts.W->rows;
    p.out_scale = 1.f;
    p.row_tiles = p.part[0].row_tiles;
    p.n_tiles = 1;
    p.splits = 1;
    p.kb_per_split = p.part[0].k_blocks;
    p.status = ws.status;
    p.gated = experts.act != nullptr ? 1 + experts.act->kind : 0;
    p.bf16 = experts.W->bf16 ? 1 : 0;
    p.n_groups = 1;
    p.experts = experts.experts;
    p.offsets = experts.offsets;
    launch_hg_width(bn, *tw[0], tx[0], *tw[1], tx[1], p, std::min(device_sm_count(), most_items), s);
}

namespace {
int launch_hgemm_any(const HalfWeight& W, const __half* xh, int T, float* y, int ldy, float out_scale, float softcap,
                     const HgemmScratch& ws, cudaStream_t s, int max_splits, const GatedAct* act, __half* yh, int ldyh,
                     const MatmulScatter* scatter) {
    if (T <= 0) return 1;
    if (!W.ready) throw std::runtime_error("launch_hgemm_tc: the f16 image of the matrix was not built");
    if (xh == nullptr) throw std::runtime_error("launch_hgemm_tc: f16 activations missing");
    if (out_scale != 1.0f || softcap != 0.f || ws.partial == nullptr) max_splits = 1;
    HgemmPlan pl = hgemm_tc_plan(W.rows, W.cols, T, max_splits);
    if (pl.splits > 1 && pl.partial_floats > ws.partial_floats) {
        pl.splits = 1;
        pl.kb_per_split = (int)(W.cols / HG_BK);
    }
    alignas(64) CUtensorMap tx;
    encode_half_matrix(&tx, xh, (int64_t)T * W.n_groups, W.cols, pl.bn, W.bf16);
    HgParams p{};
    p.T = T;
    p.K = (int)W.cols;
    p.rows = (int)W.rows;
    p.part[0].y = y;
    p.part[0].ldy = ldy;
    p.part[0].yh = yh;
    p.part[0].ldyh = ldyh;
    if (act != nullptr) {
        p.part[0].act_limit = act->limit;
        p.part[0].act_pre = act->pre;
        p.part[0].act_post = act->post;
    }
    p.out_scale = out_scale;
    p.softcap = softcap;
    p.row_tiles = pl.row_tiles;
    p.n_tiles = pl.n_tiles;
    p.splits = pl.splits;
    p.kb_per_split = pl.kb_per_split;
    p.partial = ws.partial;
    p.status = ws.status;
    p.gated = act != nullptr ? 1 + act->kind : 0;
    p.bf16 = W.bf16 ? 1 : 0;
    p.n_groups = W.n_groups;
    for (int g = 0; g < kMaxRowGroups; ++g) p.group_end[g] = W.group_end[g];
    p.group_tiles = W.group_tiles;
    p.scattered = scatter != nullptr ? 1 : 0;
    if (scatter != nullptr) p.scatter = *scatter;
    const int grid = std::min(device_sm_count(), p.row_tiles * p.n_tiles * p.splits);
    const CUtensorMap& tw = *reinterpret_cast<const CUtensorMap*>(W.tmap);
    launch_hg_width(pl.bn, tw, tx, tw, tx, p, grid, s);
    return pl.splits;
}
}  // namespace

}  // namespace mk
