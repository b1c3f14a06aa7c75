// Warp-level bf16 mma.sync m16n8k16 fragments and cp.async, shared by the chunk-wise linear-attention kernels.
#pragma once
#include "common.cuh"

#ifdef __CUDACC__

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
  const int sz = valid ? 16 : 0;  // 0: nothing is read, the 16 bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(sz) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// A fragment (16 x 16) of a row-major [m][k] matrix.
__device__ __forceinline__ void frag_a(const bf16* s, int ld, int m0, int k0, int lane, uint32_t* a) {
  const int row = m0 + (lane & 7) + ((lane >> 3) & 1) * 8, col = k0 + (lane >> 4) * 8;
  ldsm_x4(smem_u32(s + row * ld + col), a[0], a[1], a[2], a[3]);
}
// A fragment (16 x 16) of A[m][k] stored as [k][m].
__device__ __forceinline__ void frag_a_t(const bf16* s, int ld, int m0, int k0, int lane, uint32_t* a) {
  const int row = k0 + (lane & 7) + (lane >> 4) * 8, col = m0 + ((lane >> 3) & 1) * 8;
  ldsm_x4_t(smem_u32(s + row * ld + col), a[0], a[1], a[2], a[3]);
}
// B fragments of two 8-wide n-tiles (n0, n0 + 8) over 16 k, B[k][n] stored as [n][k].
__device__ __forceinline__ void frag_b_nk(const bf16* s, int ld, int n0, int k0, int lane, uint32_t* b) {
  const int j = lane >> 3, r = lane & 7;
  const int row = n0 + (j >> 1) * 8 + r, col = k0 + (j & 1) * 8;
  ldsm_x4(smem_u32(s + row * ld + col), b[0], b[1], b[2], b[3]);
}
// Same, B[k][n] stored as [k][n].
__device__ __forceinline__ void frag_b_kn(const bf16* s, int ld, int k0, int n0, int lane, uint32_t* b) {
  const int j = lane >> 3, r = lane & 7;
  const int row = k0 + (j & 1) * 8 + r, col = n0 + (j >> 1) * 8;
  ldsm_x4_t(smem_u32(s + row * ld + col), b[0], b[1], b[2], b[3]);
}

#endif  // __CUDACC__
