// How rows travel between the matmuls and the kernels around them.
#pragma once
#include "common.cuh"
#include <cuda_bf16.h>

namespace mk {

// A matmul's f32 output [rows][ld], possibly still cut into n partial sums (split-K) `stride` floats apart, which the consumer
// adds in index order.
struct Shares {
    const float* p = nullptr;
    int n = 1;
    int64_t stride = 0;
    int ld = 0;
#ifdef __CUDACC__
    __device__ __forceinline__ float at(int64_t row, int col) const {
        const float* q = p + row * ld + col;
        float v = *q;
#pragma unroll 4
        for (int s = 1; s < n; ++s) v += q[s * stride];
        return v;
    }
    __device__ __forceinline__ float4 at4(int64_t row, int col) const {  // col, ld and stride multiples of 4
        const float* q = p + row * ld + col;
        float4 v = *reinterpret_cast<const float4*>(q);
#pragma unroll 4
        for (int s = 1; s < n; ++s) {
            const float4 w = *reinterpret_cast<const float4*>(q + s * stride);
            v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
        }
        return v;
    }
#endif
};

// A matmul's input rows [rows][ld]: bfloat16 (h) or f32 (f), whichever is set.  Columns from the matrix's true width up to end()
// are zeros, written by the kernel that makes the rows.  A row may be made of parts with an image each (part()), one after the
// other.
struct RowImage {
    __nv_bfloat16* h = nullptr;
    float* f = nullptr;
    int ld = 0;
    int cols = 0;  // columns of this part, 0: the whole row
    __host__ __device__ int end() const { return cols > 0 ? cols : ld; }
    RowImage part(int first, int n) const {
        RowImage r = *this;
        if (r.h != nullptr) r.h += first;
        if (r.f != nullptr) r.f += first;
        r.cols = n;
        return r;
    }
#ifdef __CUDACC__
    __device__ __forceinline__ bool any() const { return h != nullptr || f != nullptr; }
    __device__ __forceinline__ void put(int64_t row, int col, float v) const {
        if (h != nullptr) h[row * ld + col] = __float2bfloat16_rn(v);
        else f[row * ld + col] = v;
    }
    __device__ __forceinline__ void put4(int64_t row, int col, float4 v) const {  // col and ld multiples of 4
        if (h != nullptr) {
            __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
            *reinterpret_cast<uint2*>(h + row * ld + col) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
        } else {
            *reinterpret_cast<float4*>(f + row * ld + col) = v;
        }
    }
#endif
};

// A tick's lanes as the recurrent kernels see them: the slot half to read (-1: zeros), the half to write, and the packed rows.
// Staged by the host, so a kernel may read it before its predecessor has finished.
struct StateLane {
    int32_t in, out, first, n;
};
struct StateLanes {
    const StateLane* lane = nullptr;  // [lanes], 16-byte aligned
    int lanes = 0;
#ifdef __CUDACC__
    __device__ __forceinline__ StateLane at(int i) const {
        const int4 v = reinterpret_cast<const int4*>(lane)[i];
        return StateLane{v.x, v.y, v.z, v.w};
    }
#endif
};

// How a gated feed-forward joins its gate and up sums.
//   Silu: silu(g) * u.  GeluTanh: gelu(g) * u.
//   Clamped: g and u times `pre` of the row (the weight of a mixture of experts, which multiplies the expert's input), held within
//   `limit` (g from above only), g * sigmoid(1.702 g) * (u + 1), times `post` of the row (the gate of a shared expert).
struct GatedAct {
    enum Kind : int { Silu = 0, GeluTanh = 1, Clamped = 2 };
    int kind = Silu;
    float limit = 0.f;
    const float* pre = nullptr;   // [rows], null: 1
    const float* post = nullptr;  // [rows], null: 1
};

#ifdef __CUDACC__
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float clamped_gate_f(float g, float u, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoid_f(1.702f * g) * (u + 1.0f);
}
__device__ __forceinline__ float gelu_tanh_f(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }
#endif

}  // namespace mk
