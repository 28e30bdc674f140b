// bf16 operands of mma.sync m16n8k16 on row-major tiles in shared memory: asynchronous copies, fragment
// loads and addresses, and the split of an f32 value into two bf16 planes.  Row strides in elements; a row
// starts on 16 bytes.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace tlb {

#ifdef __CUDACC__

__device__ __forceinline__ void rc_cp16(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}
__device__ __forceinline__ void rc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void rc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void rc_ldm(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void rc_ldmt(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void rc_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two f32 values as bf16 planes: hi, and lo = what hi leaves out
__device__ __forceinline__ void rc_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  hi = *(const uint32_t*)&h;
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
  lo = *(const uint32_t*)&l;
}
// fragment addresses: A from [row][k]; B from [n][k]; B from [k][n]; A from [k][row]
__device__ __forceinline__ const __nv_bfloat16* rc_a(const __nv_bfloat16* s, int ld, int r, int k, int lane) {
  return s + (r + (lane & 15)) * ld + k + (lane >> 4) * 8;
}
__device__ __forceinline__ const __nv_bfloat16* rc_bn(const __nv_bfloat16* s, int ld, int n, int k, int lane) {
  return s + (n + (lane & 7) + ((lane >> 4) << 3)) * ld + k + ((lane >> 3) & 1) * 8;
}
__device__ __forceinline__ const __nv_bfloat16* rc_bk(const __nv_bfloat16* s, int ld, int k, int n, int lane) {
  return s + (k + (lane & 15)) * ld + n + (lane >> 4) * 8;
}
__device__ __forceinline__ const __nv_bfloat16* rc_at(const __nv_bfloat16* s, int ld, int r, int k, int lane) {
  return s + (k + ((lane >> 4) << 3) + (lane & 7)) * ld + r + ((lane >> 3) & 1) * 8;
}

#endif  // __CUDACC__

}  // namespace tlb
