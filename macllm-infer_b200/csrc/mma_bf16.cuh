// Warp-level bfloat16 products (m16n8k16, f32 accumulators) out of shared memory, and f32 numbers as sums of bfloat16 ones.
#pragma once
#include "common.cuh"
#include <cuda_bf16.h>

namespace mk {

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
__device__ __forceinline__ void mc_cp_async16(void* dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;  // 0: the 16 bytes become zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(mc_smem(dst)), "l"(src), "r"(bytes) : "memory");
}
// x and y as bfloat16 numbers, and what that left of them.
__device__ __forceinline__ void mc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// Fragments of operands that lie in shared memory, rows `pitch` bfloat16 numbers apart (a multiple of 8), from `p` on.
// A, 16 rows x 16 inner indices: stored [row][inner], or [inner][row].
__device__ __forceinline__ void mma_a(uint32_t (&r)[4], const __nv_bfloat16* p, int pitch, int lane) { mc_ldmatrix(r, p + (lane & 15) * pitch + (lane >> 4) * 8); }
__device__ __forceinline__ void mma_a_t(uint32_t (&r)[4], const __nv_bfloat16* p, int pitch, int lane) {
    mc_ldmatrix_t(r, p + ((lane >> 4) * 8 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 8);
}
// B, 16 inner indices x 16 columns (two tiles: r[0], r[1] and r[2], r[3]): stored [column][inner], or [inner][column].
__device__ __forceinline__ void mma_b(uint32_t (&r)[4], const __nv_bfloat16* p, int pitch, int lane) {
    mc_ldmatrix(r, p + ((lane & 7) + (lane >> 4) * 8) * pitch + ((lane >> 3) & 1) * 8);
}
__device__ __forceinline__ void mma_b_t(uint32_t (&r)[4], const __nv_bfloat16* p, int pitch, int lane) {
    mc_ldmatrix_t(r, p + ((lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (lane >> 4) * 8);
}
// A matrix held as the sum of two: the high part, and `rest` numbers further on what that left.
struct Split {
    __nv_bfloat16* p = nullptr;
    int pitch = 0, rest = 0;
    __device__ __forceinline__ __nv_bfloat16* at(int row, int col) const { return p + row * pitch + col; }
    __device__ __forceinline__ void put2(int row, int col, float x, float y) const {  // col even
        uint32_t hi, lo;
        mc_split(x, y, hi, lo);
        *reinterpret_cast<uint32_t*>(at(row, col)) = hi;
        *reinterpret_cast<uint32_t*>(at(row, col) + rest) = lo;
    }
    __device__ __forceinline__ float2 get2(int row, int col) const {
        const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(at(row, col)));
        const float2 l = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(at(row, col) + rest));
        return make_float2(h.x + l.x, h.y + l.y);
    }
};
// acc (two tiles) += A B for split operands, the product of both rests left out.
__device__ __forceinline__ void mma_split(float (&c0)[4], float (&c1)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[4], const uint32_t (&bl)[4]) {
    mc_mma(c0, ah, bh[0], bh[1]);
    mc_mma(c1, ah, bh[2], bh[3]);
    mc_mma(c0, ah, bl[0], bl[1]);
    mc_mma(c1, ah, bl[2], bl[3]);
    mc_mma(c0, al, bh[0], bh[1]);
    mc_mma(c1, al, bh[2], bh[3]);
}

}  // namespace mk
