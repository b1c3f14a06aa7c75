// Pieces shared by the tcgen05 prefill attention kernels (attention_tc.cu, mla_prefill.cu): descriptors, tensor-memory
// access, the softmax of one 64-key tile, tensor maps.
#pragma once
#include <type_traits>
#include "common.cuh"

#include <cuda.h>

#include <mutex>

namespace {

constexpr int BQ2 = 256;           // query rows per CTA of the two-group kernels
constexpr int BKV2 = 64;           // keys per tile of the head-dim-256 and latent kernels
constexpr int GROUPS = 2;          // query tiles of 128 rows per CTA; their softmax groups alternate on the tensor core
constexpr int THREADS = 64 + GROUPS * 128;
constexpr float RESCALE_LOG2 = 8.f;  // O and the row sum move to a new maximum only when it grew by more than 2^8

struct TcSmem {
  uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[GROUPS], p_ready[GROUPS], o_full[GROUPS];
  uint32_t tmem_slot;
  int abort_flag;
};

// MN-major operand (rows = contraction index, 128-byte rows of 64 consecutive N elements, 128-byte swizzle):
// `lbo` = byte stride between blocks of 64 N elements, `sbo` = byte stride between groups of 8 contraction rows.
__device__ __forceinline__ uint64_t umma_desc_mn_sw128(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFFu) >> 4);
  d |= (uint64_t)((lbo >> 4) & 0x3FFFu) << 16;
  d |= (uint64_t)((sbo >> 4) & 0x3FFFu) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}
// bf16 x bf16 -> f32, A K-major, B K-major or MN-major
__host__ __device__ constexpr uint32_t idesc_bf16(uint32_t m, uint32_t n, uint32_t b_mn_major) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn_major << 16) | ((n >> 3) << 17) | ((m >> 4) << 24);
}

__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t* r) {
  tmem_ld16(taddr, r);
  tmem_ld16(taddr + 16, r + 16);
}
// Each thread of the warp writes 16 consecutive 32-bit columns of its own TMEM lane.
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]),
        "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// D[tmem] (+)= A[tmem] * B[smem]: A is a 128-row matrix in tensor memory (row = lane, two bf16 per 32-bit column).
__device__ __forceinline__ void umma_bf16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ float max3(float a, float b, float c) {
  float y;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(y) : "f"(a), "f"(b), "f"(c));
  return y;
}
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// One tile of 64 keys for one query row per thread (the head-dim-256 and MLA kernels): S of the tile -> registers ->
// maximum -> lazy rescale of O (`o_cols` columns at `o_row`) -> P as bf16 over the first 32 columns of S -> `p_ready`.
// `o_full` / `o_parity` name the completion of the previous product into the same O (ignored for j == 0).
template <bool MASK>
__device__ __forceinline__ bool softmax_tile64(uint64_t* s_full, uint32_t s_parity, uint32_t s_row, uint32_t o_row, int o_cols, uint64_t* o_full, uint32_t o_parity, int j, int limit, int lo,
                                               float scale_log2, float& m, float& l, uint64_t* p_ready, int lane, volatile int* abort_flag) {
  if (!mbar_wait(s_full, s_parity, abort_flag)) return false;
  tc_fence_after();
  uint32_t v[BKV2];
  tmem_ld32(s_row, v);
  tmem_ld32(s_row + 32, v + 32);
  tmem_ld_wait();
  float mx_raw;
  if constexpr (MASK) {
    mx_raw = -INFINITY;
#pragma unroll
    for (int i = 0; i < BKV2; ++i)
      if (i <= limit && i > lo) mx_raw = fmaxf(mx_raw, __uint_as_float(v[i]));
  } else {
    float m0 = max3(__uint_as_float(v[0]), __uint_as_float(v[1]), __uint_as_float(v[2]));
    float m1 = max3(__uint_as_float(v[3]), __uint_as_float(v[4]), __uint_as_float(v[5]));
    float m2 = max3(__uint_as_float(v[6]), __uint_as_float(v[7]), __uint_as_float(v[8]));
    float m3 = max3(__uint_as_float(v[9]), __uint_as_float(v[10]), __uint_as_float(v[11]));
#pragma unroll
    for (int i = 12; i + 7 < BKV2; i += 8) {
      m0 = max3(m0, __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
      m1 = max3(m1, __uint_as_float(v[i + 2]), __uint_as_float(v[i + 3]));
      m2 = max3(m2, __uint_as_float(v[i + 4]), __uint_as_float(v[i + 5]));
      m3 = max3(m3, __uint_as_float(v[i + 6]), __uint_as_float(v[i + 7]));
    }
    // 12 + 8 * 6 = 60: four columns left
    m0 = max3(m0, __uint_as_float(v[60]), __uint_as_float(v[61]));
    m1 = max3(m1, __uint_as_float(v[62]), __uint_as_float(v[63]));
    mx_raw = fmaxf(max3(m0, m1, m2), m3);
  }
  const float mx = mx_raw * scale_log2;
  // the previous product must be complete before O is rescaled
  if (j >= 1) {
    if (!mbar_wait(o_full, o_parity, abort_flag)) return false;
    tc_fence_after();
  }
  float alpha = 1.f;
  if (mx > m + RESCALE_LOG2 || (m == -INFINITY && mx > -INFINITY)) {
    alpha = (m == -INFINITY) ? 0.f : ex2_approx(m - mx);
    m = mx;
  }
  if (j >= 1 && __any_sync(0xFFFFFFFFu, alpha != 1.f)) {
    const float2 a2 = make_float2(alpha, alpha);
#pragma unroll 1
    for (int c = 0; c < o_cols; c += 32) {
      uint32_t w[32];
      tmem_ld32(o_row + c, w);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; i += 2) {
        const float2 t2 = __fmul2_rn(make_float2(__uint_as_float(w[i]), __uint_as_float(w[i + 1])), a2);
        w[i] = __float_as_uint(t2.x);
        w[i + 1] = __float_as_uint(t2.y);
      }
      tmem_st16(o_row + c, w);
      tmem_st16(o_row + c + 16, w + 16);
    }
    l *= alpha;
  }
  const float neg = (m == -INFINITY) ? 0.f : -m;
  float2 sum2 = make_float2(0.f, 0.f), sum3 = make_float2(0.f, 0.f);
  const float2 sc2 = make_float2(scale_log2, scale_log2), ng2 = make_float2(neg, neg);
#pragma unroll
  for (int c = 0; c < BKV2; c += 32) {
    uint32_t packed[16];
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      const float2 t2 = __ffma2_rn(make_float2(__uint_as_float(v[c + i]), __uint_as_float(v[c + i + 1])), sc2, ng2);
      const float2 t3 = __ffma2_rn(make_float2(__uint_as_float(v[c + i + 2]), __uint_as_float(v[c + i + 3])), sc2, ng2);
      float2 e = make_float2(ex2_approx(t2.x), ex2_approx(t2.y));
      float2 f = make_float2(ex2_approx(t3.x), ex2_approx(t3.y));
      if constexpr (MASK) {
        if (c + i > limit || c + i <= lo) e.x = 0.f;
        if (c + i + 1 > limit || c + i + 1 <= lo) e.y = 0.f;
        if (c + i + 2 > limit || c + i + 2 <= lo) f.x = 0.f;
        if (c + i + 3 > limit || c + i + 3 <= lo) f.y = 0.f;
      }
      sum2 = __fadd2_rn(sum2, e);
      sum3 = __fadd2_rn(sum3, f);
      const bf162 pe = __floats2bfloat162_rn(e.x, e.y), pf = __floats2bfloat162_rn(f.x, f.y);
      packed[i >> 1] = *reinterpret_cast<const uint32_t*>(&pe);
      packed[(i >> 1) + 1] = *reinterpret_cast<const uint32_t*>(&pf);
    }
    tmem_st16(s_row + (c >> 1), packed);
  }
  sum2 = __fadd2_rn(sum2, sum3);
  tmem_st_wait();
  l += sum2.x + sum2.y;
  tc_fence_before();
  __syncwarp();
  if (lane == 0) mbar_arrive(p_ready);
  return true;
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*, const cuuint32_t*,
                                  CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiledFn get_encode_attn() {
  static EncodeTiledFn fn = nullptr;
  static std::once_flag once;
  std::call_once(once, [] {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeTiledFn>(p);
  });
  return fn;
}

// [rows, heads, dim] bf16, contiguous; box = 64 columns x 1 head x box_rows rows, 128-byte swizzle
[[maybe_unused]] int make_tmap_rows_heads(CUtensorMap* out, const void* ptr, long long rows, int heads, int box_rows, int dim) {
  EncodeTiledFn enc = get_encode_attn();
  PG_REQUIRE(enc != nullptr, "cuTensorMapEncodeTiled is not available from this driver");
  PG_REQUIRE(((uintptr_t)ptr & 15) == 0, "TMA base address must be 16-byte aligned");
  cuuint64_t dims[3] = {(cuuint64_t)dim, (cuuint64_t)heads, (cuuint64_t)rows};
  cuuint64_t strides[2] = {(cuuint64_t)dim * 2, (cuuint64_t)heads * dim * 2};
  cuuint32_t box[3] = {64u, 1u, (cuuint32_t)box_rows};
  cuuint32_t estr[3] = {1, 1, 1};
  CUresult r = enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                   CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  PG_REQUIRE(r == CUDA_SUCCESS, "cuTensorMapEncodeTiled failed with code %d", (int)r);
  return PG_OK;
}


// generic tiled tensor map over bf16 with the 128-byte swizzle (inner box = 64 elements)
[[maybe_unused]] int make_tmap_bf16(CUtensorMap* out, const void* ptr, int rank, const cuuint64_t* dims, const cuuint64_t* strides_bytes, const cuuint32_t* box) {
  EncodeTiledFn enc = get_encode_attn();
  PG_REQUIRE(enc != nullptr, "cuTensorMapEncodeTiled is not available from this driver");
  PG_REQUIRE(((uintptr_t)ptr & 15) == 0, "TMA base address must be 16-byte aligned");
  for (int i = 0; i + 1 < rank; ++i) PG_REQUIRE(strides_bytes[i] % 16 == 0, "TMA stride %d of %llu bytes is not a multiple of 16", i, (unsigned long long)strides_bytes[i]);
  cuuint32_t estr[5] = {1, 1, 1, 1, 1};
  CUresult r = enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (cuuint32_t)rank, const_cast<void*>(ptr), dims, strides_bytes, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  PG_REQUIRE(r == CUDA_SUCCESS, "cuTensorMapEncodeTiled failed with code %d", (int)r);
  return PG_OK;
}

}  // namespace
