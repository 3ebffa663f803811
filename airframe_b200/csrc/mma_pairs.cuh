// Tensor-core products (mma.sync, bfloat16 operands, 32-bit sums) whose operands are 32-bit values in two parts: a value
// is hi + lo, both bfloat16, and a product is hi hi + hi lo + lo hi (16 to 17 bits of mantissa; what is dropped is lo lo).
// For recurrences, whose states, keys and weights a design wants in 32 bits.
#pragma once
#include "common.cuh"

__device__ __forceinline__ uint32_t mp_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mp_ldm4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mp_smem(p)) : "memory");
}
__device__ __forceinline__ void mp_ldm4t(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mp_smem(p)) : "memory");
}
__device__ __forceinline__ void mp_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
               "{%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// hi + lo: two neighbours packed as bfloat16
__device__ __forceinline__ void mp_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ void mp_put4(__nv_bfloat16* hi, __nv_bfloat16* lo, const float* y) {
  uint32_t h0, l0, h1, l1;
  mp_split2(y[0], y[1], h0, l0);
  mp_split2(y[2], y[3], h1, l1);
  *reinterpret_cast<uint2*>(hi) = make_uint2(h0, h1);
  *reinterpret_cast<uint2*>(lo) = make_uint2(l0, l1);
}
// 16 bytes from global to shared memory without a register in between (`on` false: zeros)
__device__ __forceinline__ void mp_cp16(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(mp_smem(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}
__device__ __forceinline__ void mp_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void mp_cp_wait() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
