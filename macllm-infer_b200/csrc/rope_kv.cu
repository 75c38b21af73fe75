// Fused per-head QK RMSNorm + half-split RoPE + paged-KV scatter.
//
// Replaces, per layer, SelfAttention::project_packed_qkv's per-head norms (src/decoder.rs:1137-1154,
// applied BEFORE the rotation), RotaryEmbedding::apply (src/decoder.rs:203-257, half-split layout on
// the first rotary_dim dims) and PagedKvBatchReservation::write_layer
// (crates/macllm-kv/src/cache.rs:2543-2643): K is stored after the rotation, V unmodified, both at
// KV-head cardinality, token at slot block*block_tokens + row.
// One warp per (token, head); the head vector is staged in shared memory so any head_dim works.
#include "kernels.h"
#include "rope_head.cuh"
#include <algorithm>

namespace mk {

namespace {

constexpr int RK_WARPS = 4;

template <typename KV>
__device__ __forceinline__ KV to_kv(float v);
template <>
__device__ __forceinline__ float to_kv<float>(float v) { return v; }
template <>
__device__ __forceinline__ __half to_kv<__half>(float v) { return __float2half_rn(v); }

template <typename KV>
__global__ void __launch_bounds__(RK_WARPS * 32) rope_kv_kernel(RopeKvArgs a) {
    __shared__ float buf[RK_WARPS][RK_MAX_D];
    pdl_trigger();
    pdl_wait();
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int heads_total = a.q_heads + 2 * a.kv_heads;
    int head = blockIdx.y * RK_WARPS + warp;
    int t = blockIdx.x;
    if (head >= heads_total) return;
    const int d = rope_row_width(a);
    float* x = buf[warp];

    int kind, hh;  // 0 = q, 1 = k, 2 = v
    if (head < a.q_heads) { kind = 0; hh = head; }
    else if (head < a.q_heads + a.kv_heads) { kind = 1; hh = head - a.q_heads; }
    else { kind = 2; hh = head - a.q_heads - a.kv_heads; }
    rope_head_prepare(a, kind, hh, t, kind != 2 && a.cos_t != nullptr ? a.positions[t] : 0, x, lane);
    if (kind == 0) {
        float* dst = a.q_out != nullptr ? a.q_out + (int64_t)t * a.ldq_out + hh * d : a.q + (int64_t)t * a.ldq + hh * d;
        for (int i = lane; i < d; i += 32) dst[i] = x[i];
    } else {
        int64_t slot = a.slots[t];
        int64_t blk = slot / a.block_tokens, row = slot % a.block_tokens;
        int64_t base = ((kv_page_index(blk, a.layer, a.layers, a.pool_blocks) * a.kv_heads + hh) * a.block_tokens + row) * (int64_t)d;
        KV* pool = reinterpret_cast<KV*>(kind == 1 ? a.k_pool : a.v_pool);
        for (int i = lane; i < d; i += 32) pool[base + i] = to_kv<KV>(x[i]);
    }
}

// One CTA per token: all heads of the token in shared memory ((q_heads + kv_heads) * d + kv_heads * dv floats).
// vec: every row starts on 16 bytes and head widths are multiples of four.
template <typename KV, int THREADS>
__global__ void __launch_bounds__(THREADS) rope_kv_rows_kernel(RopeKvArgs a, int vec) {
    extern __shared__ __align__(16) float rr_row[];
    __shared__ float red[2][32];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, dv = a.dv > 0 ? a.dv : a.d, D = rope_row_width(a);
    const int qw = a.q_heads * a.d, kw = a.kv_heads * a.d, vw = a.kv_heads * dv;
    float *xq = rr_row, *xk = xq + qw, *xv = xk + kw;
    // a projection's row: the shares' sum and the bias; returns the thread's sum of squares
    auto load = [&](float* dst, const float* src, int n, int parts, int64_t stride, const float* bias) {
        float ss = 0.f;
        if (vec) {
            for (int c = threadIdx.x * 4; c < n; c += THREADS * 4) {
                float4 v = *reinterpret_cast<const float4*>(src + c);
#pragma unroll 8
                for (int p = 1; p < parts; ++p) {
                    const float4 w = *reinterpret_cast<const float4*>(src + (int64_t)p * stride + c);
                    v = make_float4(v.x + w.x, v.y + w.y, v.z + w.z, v.w + w.w);
                }
                if (bias != nullptr) {
                    const float4 b = *reinterpret_cast<const float4*>(bias + c);
                    v = make_float4(v.x + b.x, v.y + b.y, v.z + b.z, v.w + b.w);
                }
                *reinterpret_cast<float4*>(dst + c) = v;
                ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
            }
            return ss;
        }
        for (int c = threadIdx.x; c < n; c += THREADS) {
            float v = src[c];
            for (int p = 1; p < parts; ++p) v += src[(int64_t)p * stride + c];
            if (bias != nullptr) v += bias[c];
            dst[c] = v;
            ss = fmaf(v, v, ss);
        }
        return ss;
    };
    float sq = load(xq, a.q + (int64_t)t * a.ldq, qw, a.qk_splits, a.qk_split_stride, a.q_bias);
    float sk = load(xk, a.k + (int64_t)t * a.ldk, kw, a.qk_splits, a.qk_split_stride, a.k_bias);
    load(xv, a.v + (int64_t)t * a.ldv, vw, a.v_splits, a.v_split_stride, a.v_bias);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) {
        red[0][threadIdx.x >> 5] = sq;
        red[1][threadIdx.x >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) {
        sq += red[0][w];
        sk += red[1][w];
    }
    const float rq = sqrtf(sq / (float)qw + a.norm_eps), rk = sqrtf(sk / (float)kw + a.norm_eps);
    const int rd = a.cos_t != nullptr ? a.rotary_dim : 0, half = rd / 2;
    const float* cs = a.cos_t + (rd > 0 ? (int64_t)a.positions[t] * half : 0);
    const float* sn = a.sin_t + (rd > 0 ? (int64_t)a.positions[t] * half : 0);
    // value c of the head at x (norm weights at w): normed, then turned with its partner
    auto turned = [&](const float* x, const float* w, float root, int c) {
        const float own = x[c] / root * w[c];
        if (c >= rd) return own;
        const int i = a.interleaved ? c >> 1 : (c < half ? c : c - half);
        const bool first = a.interleaved ? (c & 1) == 0 : c < half;
        const int p = a.interleaved ? c ^ 1 : (first ? c + half : c - half);
        const float other = x[p] / root * w[p];
        return first ? own * cs[i] - other * sn[i] : own * cs[i] + other * sn[i];
    };
    float* q_out = a.q_out + (int64_t)t * a.ldq_out;
#pragma unroll 4
    for (int i = threadIdx.x; i < a.q_heads * D; i += THREADS) {
        const int h = i / D, c = i - h * D;
        q_out[i] = c < a.d ? turned(xq + h * a.d, a.q_norm_w + h * a.d, rq, c) : 0.f;
    }
    const int64_t slot = a.slots[t], blk = slot / a.block_tokens, row = slot % a.block_tokens;
    KV *kp = reinterpret_cast<KV*>(a.k_pool), *vp = reinterpret_cast<KV*>(a.v_pool);
    const int64_t page = kv_page_index(blk, a.layer, a.layers, a.pool_blocks) * a.kv_heads;
#pragma unroll 2
    for (int i = threadIdx.x; i < a.kv_heads * D; i += THREADS) {
        const int h = i / D, c = i - h * D;
        const int64_t at = ((page + h) * a.block_tokens + row) * (int64_t)D + c;
        kp[at] = to_kv<KV>(c < a.d ? turned(xk + h * a.d, a.k_norm_w + h * a.d, rk, c) : 0.f);
        vp[at] = to_kv<KV>(c < dv ? xv[h * dv + c] : 0.f);
    }
}

template <typename KV, int THREADS>
void launch_rope_rows(const RopeKvArgs& a, size_t smem, int vec, cudaStream_t s) {
    auto* kernel = rope_kv_rows_kernel<KV, THREADS>;
    ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), smem);
    launch_pdl(kernel, dim3((unsigned)a.T), dim3(THREADS), smem, s, a, vec);
}

template <typename KV>
__global__ void cow_copy_kernel(KV* k_pool, KV* v_pool, int64_t src_block, int64_t dst_block, int rows, int layers, int64_t pool_blocks,
                                int kv_heads, int block_tokens, int d) {
    // one CTA per (layer, kv_head)
    int layer = blockIdx.x / kv_heads, h = blockIdx.x % kv_heads;
    int64_t s = ((kv_page_index(src_block, layer, layers, pool_blocks) * kv_heads + h) * block_tokens) * (int64_t)d;
    int64_t t = ((kv_page_index(dst_block, layer, layers, pool_blocks) * kv_heads + h) * block_tokens) * (int64_t)d;
    for (int i = threadIdx.x; i < rows * d; i += blockDim.x) {
        k_pool[t + i] = k_pool[s + i];
        v_pool[t + i] = v_pool[s + i];
    }
}

}  // namespace

void launch_rope_kv(const RopeKvArgs& a, cudaStream_t s) {
    if (a.T <= 0) return;
    if (std::max({a.d, a.dv, a.d_row}) > RK_MAX_D) throw std::runtime_error("launch_rope_kv: head_dim above 256 is not supported");
    if (a.d_row > 0 && (a.d_row < a.d || a.d_row < a.dv || a.q_out == nullptr))
        throw std::runtime_error("launch_rope_kv: padded heads need a separate query output at least as wide as the heads");
    int heads_total = a.q_heads + 2 * a.kv_heads;
    dim3 grid((unsigned)a.T, (unsigned)((heads_total + RK_WARPS - 1) / RK_WARPS));
    if (a.kv_f16)
        launch_pdl(rope_kv_kernel<__half>, grid, dim3(RK_WARPS * 32), 0, s, a);
    else
        launch_pdl(rope_kv_kernel<float>, grid, dim3(RK_WARPS * 32), 0, s, a);
    MK_LAUNCH_CHECK();
}

void launch_rope_kv_rows(const RopeKvArgs& a, cudaStream_t s) {
    if (a.T <= 0) return;
    if (a.q_out == nullptr || a.q_norm_w == nullptr || a.k_norm_w == nullptr) throw std::runtime_error("launch_rope_kv_rows: needs norm weights and a query output");
    const size_t smem = ((size_t)a.q_heads * a.d + (size_t)a.kv_heads * (a.d + (a.dv > 0 ? a.dv : a.d))) * 4;
    if (smem > (size_t)200 * 1024) throw std::runtime_error("launch_rope_kv_rows: the projections are too wide");
    const int dv = a.dv > 0 ? a.dv : a.d;
    auto on16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const int vec = a.d % 4 == 0 && dv % 4 == 0 && a.ldq % 4 == 0 && a.ldk % 4 == 0 && a.ldv % 4 == 0 && a.qk_split_stride % 4 == 0 && a.v_split_stride % 4 == 0 &&
                    on16(a.q) && on16(a.k) && on16(a.v) && on16(a.q_bias) && on16(a.k_bias) && on16(a.v_bias) ? 1 : 0;
    // ticks of a few rows: a row's latency counts, so many threads share it
    if (a.T <= 148) {
        if (a.kv_f16) launch_rope_rows<__half, 1024>(a, smem, vec, s);
        else launch_rope_rows<float, 1024>(a, smem, vec, s);
    } else {
        if (a.kv_f16) launch_rope_rows<__half, 256>(a, smem, vec, s);
        else launch_rope_rows<float, 256>(a, smem, vec, s);
    }
    MK_LAUNCH_CHECK();
}

void launch_cow_copy(void* k_pool, void* v_pool, int kv_f16, int64_t src_block, int64_t dst_block, int rows, int layers,
                     int64_t pool_blocks, int kv_heads, int block_tokens, int d, cudaStream_t s) {
    if (rows <= 0) return;
    unsigned grid = (unsigned)(layers * kv_heads);
    if (kv_f16)
        cow_copy_kernel<__half><<<grid, 128, 0, s>>>((__half*)k_pool, (__half*)v_pool, src_block, dst_block, rows,
                                                     layers, pool_blocks, kv_heads, block_tokens, d);
    else
        cow_copy_kernel<float><<<grid, 128, 0, s>>>((float*)k_pool, (float*)v_pool, src_block, dst_block, rows, layers,
                                                    pool_blocks, kv_heads, block_tokens, d);
    MK_LAUNCH_CHECK();
}

}  // namespace mk
