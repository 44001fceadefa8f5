// Warp-level bf16 matrix fragments (mma.sync m16n8k16) for products too small or too dependent for a tcgen05 tile.
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

namespace forge {

#ifdef __CUDACC__
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Row-major bf16 matrix in shared memory, rows `ld` elements apart (16-byte aligned, an odd number of 16-byte pieces apart against bank
// conflicts).  Every function loads one 16 x 16 block at (r0, c0); lanes 8 j + i address row i of its quarter j.
struct SmemMat {
    uint32_t addr; int ld;
    __device__ __forceinline__ uint32_t at(int r, int c) const { return addr + uint32_t(r * ld + c) * 2; }
    // A operand, rows = M index
    __device__ __forceinline__ void a(uint32_t (&f)[4], int r0, int c0, int lane) const { ldsm4(f, at(r0 + ((lane >> 3) & 1) * 8 + (lane & 7), c0 + (lane >> 4) * 8)); }
    // A operand, rows = K index
    __device__ __forceinline__ void a_t(uint32_t (&f)[4], int k0, int m0, int lane) const { ldsm4t(f, at(k0 + (lane >> 4) * 8 + (lane & 7), m0 + ((lane >> 3) & 1) * 8)); }
    // B operand of two neighbouring N tiles ({f0, f1} and {f2, f3}), rows = N index
    __device__ __forceinline__ void b(uint32_t (&f)[4], int n0, int k0, int lane) const { ldsm4(f, at(n0 + (lane >> 4) * 8 + (lane & 7), k0 + ((lane >> 3) & 1) * 8)); }
    // the same, rows = K index
    __device__ __forceinline__ void b_t(uint32_t (&f)[4], int k0, int n0, int lane) const { ldsm4t(f, at(k0 + ((lane >> 3) & 1) * 8 + (lane & 7), n0 + (lane >> 4) * 8)); }
};

// x = hi + lo up to 2^-17 of x
__device__ __forceinline__ void split_bf16(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
    hi = __float2bfloat16_rn(x);
    lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}
__device__ __forceinline__ void split_bf16x2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
// 16 bytes from global to shared memory, or zeros
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
#endif

}  // namespace forge
