// Warp-level tensor-core helpers (mma.sync m16n8k16, BF16 operands, FP32 sums), matrix loads from
// shared memory and asynchronous copies, for the kernels whose products are too small or too
// entangled with scalar work for a tcgen05 tile.
//
// Operand addresses, lane i supplying one 16-byte row of an 8 x 8 block:
//   A [m][k]      ldsm4 (p + (m0 + (lane & 15)) * ld + k0 + (lane >> 4) * 8)
//   A from [k][m] ldsm4t(p + (k0 + (lane & 7) + (lane >> 4) * 8) * ld + m0 + ((lane >> 3) & 1) * 8)
//   B from [n][k] ldsm4 (p + (n0 + (lane & 7) + (lane >> 4) * 8) * ld + k0 + ((lane >> 3) & 1) * 8)
//   B from [k][n] ldsm4t(p + (k0 + (lane & 15)) * ld + n0 + (lane >> 4) * 8)
// (B: two column tiles of 8, words 0-1 and 2-3).  Sums: c[0..1] row lane / 4, columns 2 (lane % 4)
// and the next; c[2..3] the same columns of row lane / 4 + 8.
#pragma once
#include "dense.cuh"

namespace tllm {

__device__ __forceinline__ uint32_t sm32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const bf16* p)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(sm32(p)) : "memory");
}
__device__ __forceinline__ void ldsm2(uint32_t (&r)[2], const bf16* p)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(sm32(p)) : "memory");
}
__device__ __forceinline__ void ldsm2t(uint32_t (&r)[2], const bf16* p)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(sm32(p)) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const bf16* p)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(sm32(p)) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp16(bf16* dst, const bf16* src, bool valid)
{
    const int n = valid ? 16 : 0;       // 0: fill with zeros, nothing is read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(sm32(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// p = hi + lo with both parts BF16; two values packed per word
__device__ __forceinline__ void split2(float p0, float p1, uint32_t& hi, uint32_t& lo)
{
    const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(p0 - f.x, p1 - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

}  // namespace tllm
