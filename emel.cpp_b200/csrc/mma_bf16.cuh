// Legacy-path tensor core helpers shared by the attention kernels of layered decoders: ldmatrix, mma.sync m16n8k16
// with bf16 operands and f32 accumulators, and f32 values split into two bf16 operands (high part + remainder).
// Fragments, lane = 4g + t: A a0 (row g, k 2t..) a1 (row g+8, same k) a2 (row g, k 2t+8..) a3 (row g+8, k 2t+8..);
// B b0 (k 2t.., n g) b1 (k 2t+8.., n g); C c0,c1 (row g, n 2t..) c2,c3 (row g+8, n 2t..).
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

namespace emelb {

__device__ __forceinline__ void cp16_zfill(void* smem, const void* gmem, bool live) {
  const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void ldsm(uint32_t (&r)[4], const void* row) {
  const uint32_t addr = static_cast<uint32_t>(__cvta_generic_to_shared(row));
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_trans(uint32_t (&r)[4], const void* row) {
  const uint32_t addr = static_cast<uint32_t>(__cvta_generic_to_shared(row));
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_bf16_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two f32 values as packed bf16 high parts and packed remainders
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 b = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - b.x, y - b.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 unpack2(uint32_t w) { return make_float2(__uint_as_float(w << 16), __uint_as_float(w & 0xffff0000u)); }

}  // namespace emelb
