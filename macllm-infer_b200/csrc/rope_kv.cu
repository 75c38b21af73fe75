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

constexpr int RR_THREADS = 256;

// One CTA per token: all heads of the token in shared memory (kv_heads * (d + dv) + q_heads * d floats).
template <typename KV>
__global__ void __launch_bounds__(RR_THREADS) rope_kv_rows_kernel(RopeKvArgs a) {
    extern __shared__ __align__(16) float rr_row[];
    __shared__ float red[32];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, dv = a.dv > 0 ? a.dv : a.d, D = rope_row_width(a);
    const int qw = a.q_heads * a.d, kw = a.kv_heads * a.d, vw = a.kv_heads * dv;
    float *xq = rr_row, *xk = xq + qw, *xv = xk + kw;
    auto load = [&](float* dst, const float* src, int n, int parts, int64_t stride, const float* bias) {
        float ss = 0.f;
        for (int c = threadIdx.x; c < n; c += RR_THREADS) {
            float v = src[c];
            for (int p = 1; p < parts; ++p) v += src[(int64_t)p * stride + c];
            if (bias != nullptr) v += bias[c];
            dst[c] = v;
            ss = fmaf(v, v, ss);
        }
        return ss;
    };
    const float sq = load(xq, a.q + (int64_t)t * a.ldq, qw, a.qk_splits, a.qk_split_stride, a.q_bias);
    const float sk = load(xk, a.k + (int64_t)t * a.ldk, kw, a.qk_splits, a.qk_split_stride, a.k_bias);
    load(xv, a.v + (int64_t)t * a.ldv, vw, a.v_splits, a.v_split_stride, a.v_bias);
    const float rq = sqrtf(block_sum(sq, red) / (float)qw + a.norm_eps);
    const float rk = sqrtf(block_sum(sk, red) / (float)kw + a.norm_eps);  // its barriers also publish the rows
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
    for (int i = threadIdx.x; i < a.q_heads * D; i += RR_THREADS) {
        const int h = i / D, c = i - h * D;
        q_out[i] = c < a.d ? turned(xq + h * a.d, a.q_norm_w + h * a.d, rq, c) : 0.f;
    }
    const int64_t slot = a.slots[t], blk = slot / a.block_tokens, row = slot % a.block_tokens;
    KV *kp = reinterpret_cast<KV*>(a.k_pool), *vp = reinterpret_cast<KV*>(a.v_pool);
    for (int i = threadIdx.x; i < a.kv_heads * D; i += RR_THREADS) {
        const int h = i / D, c = i - h * D;
        const int64_t at = ((kv_page_index(blk, a.layer, a.layers, a.pool_blocks) * a.kv_heads + h) * a.block_tokens + row) * (int64_t)D + c;
        kp[at] = to_kv<KV>(c < a.d ? turned(xk + h * a.d, a.k_norm_w + h * a.d, rk, c) : 0.f);
        vp[at] = to_kv<KV>(c < dv ? xv[h * dv + c] : 0.f);
    }
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
    auto* kernel = a.kv_f16 ? rope_kv_rows_kernel<__half> : rope_kv_rows_kernel<float>;
    ensure_dynamic_smem(reinterpret_cast<const void*>(kernel), smem);
    launch_pdl(kernel, dim3((unsigned)a.T), dim3(RR_THREADS), smem, s, a);
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
