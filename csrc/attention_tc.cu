// Prefill attention on tcgen05 for sm_100a: causal GQA attention of ragged query rows over a paged KV cache,
// head dims 128 and 256 (the second kernel, further down, has its own notes).
//
// Head dim 128: one CTA owns 256 query rows of one query head as two tiles of 128 (two softmax groups) and walks the KV
// of its sequence in tiles of 128 keys that both tiles share:
//
//   S_g = Q_g K^T      tcgen05.mma, both operands K-major in shared memory (TMA, 128-byte swizzle), accumulator in TMEM
//   P_g = softmax tile four warps per group, one query row per thread: the row of S is read into registers in one round
//                      trip (maximum with three-input max, exponentials with packed f32x2 arithmetic and ex2.approx),
//                      P is written back as bf16 INTO TENSOR MEMORY over the first score columns (two values per 32-bit
//                      column).  Whether a tile needs the causal / length mask is a compile-time property of the tile
//                      body: the plain tiles carry no compare or select per element.
//   O_g += P_g V       tcgen05.mma with A = P_g read from tensor memory and V as an MN-major B operand (the cache stores
//                      keys as rows, which is what the contraction over keys needs transposed); O_g stays in TMEM for
//                      the whole walk.  It is rescaled (tcgen05.ld / multiply / tcgen05.st) only when a row's maximum
//                      grew by more than 2^8 since the value its exponentials refer to; the row sum follows the same
//                      reference, so the result is exact.
//
// Roles: warp 0 = TMA producer (Q once, then K and V tiles through the page table, two stages each; a tile is 4 x pages
// small boxes, which the 32 lanes issue side by side, with the page ids read one tile ahead), warp 1 = MMA issuer, in the
// order  P V of group a, next S of group a, P V of group b, next S of group b : while one group's softmax runs the
// tensor core has the other group's work, warps 2-5 / 6-9 = softmax groups a / b and output.
// TMEM: S / P of group g at columns 128 g, O of group g at 256 + 128 g.  The grid is one-dimensional with the query
// tile slowest and late tiles first, so the CTAs with the most keys start first on every SM.  Every wait is bounded and
// reports through the status word.
//
// Reference parity: the reference's prefill attention is FlashInfer's BatchPrefillWithPagedKVCache
// (pegainfer-kernels/csrc/shared/flashinfer_prefill.cu, hd256 instantiations in paged_attention.cu:977-1135), an
// mma.sync kernel on every architecture.
#include "attention_tc.cuh"

namespace {

constexpr int BKV = 128, D = 128;
constexpr int TILE_BYTES = 128 * D * 2;  // 32 KB: [2 blocks of 64 columns][128 rows][128 B]
constexpr int HALF_BYTES = TILE_BYTES / 2;

struct TcAttnParams {
  bf16* out;              // [T, hq * D]
  const int* q_indptr;    // [num_seqs + 1]
  const int* kv_lens;     // [num_seqs]
  const int* table;       // [num_seqs, table_stride]
  int table_stride, num_seqs, hq, hkv, page_size;
  long long num_pages;
  float scale_log2;       // softmax scale * log2(e)
  int window;             // head dim 256 and the biased form: a row sees its last `window` keys (0: all of them)
  float cap_in;           // capped form: softmax scale / cap, and scale_log2 holds cap * log2(e); 0: no cap
  const bf16* gate;       // capped form: [T, >= hq] rows of stride ld_gate whose sigmoid multiplies a head's output, or null
  long long ld_gate;
  const float* slopes;    // biased form: [hq], a (capped) score loses slope * distance; or null
  float out_scale;        // capped and biased form, on the output
  long long ld_out;       // row stride of out
  int mn_lbo_first;       // descriptor variant of the MN-major operand (1: LBO = stride between 64-column blocks)
  uint32_t* status;
};

// tanh for the soft cap of a score row.  Up to |z| = 1 (scores up to the cap) an odd polynomial of degree 13 with packed
// f32x2 arithmetic: tanh(z) / z fitted in z^2 by interpolation at Chebyshev nodes of [0, 1], relative error 1.6e-7, so that
// the special-function unit is left to the exponentials; beyond that 1 - 2 / (1 + e^2z).
__device__ __forceinline__ float2 tanh2_poly(float2 z) {
  const float2 u = __fmul2_rn(z, z);
  auto c = [](float a) { return make_float2(a, a); };
  float2 y = __ffma2_rn(u, c(0.0010455536f), c(-0.0062170699f));
  y = __ffma2_rn(u, y, c(0.02030552f));
  y = __ffma2_rn(u, y, c(-0.053465176f));
  y = __ffma2_rn(u, y, c(0.13325398f));
  y = __ffma2_rn(u, y, c(-0.33332857f));
  y = __ffma2_rn(u, y, c(0.99999994f));
  return __fmul2_rn(y, z);
}
__device__ __forceinline__ float tanh_ex2(float z) { return 1.f - __fdividef(2.f, 1.f + ex2_approx(z * 2.8853900817779268f)); }

// CAPPED: soft cap on the scores and a sigmoid gate per (token, head) on the output.  BIASED: and a sliding window (key tiles in
// front of the first row's window are skipped; tile numbers below count from j0) and a bias that grows with the distance.
enum { FORM_PLAIN = 0, FORM_CAPPED = 1, FORM_BIASED = 2 };
template <int FORM>
__global__ void __launch_bounds__(THREADS, 1) prefill_attn_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv, const TcAttnParams p) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = smem_u32(smem_raw);
  uint8_t* tiles = smem_raw + (((base + 1023u) & ~1023u) - base);
  uint8_t* q_tile = tiles;                            // GROUPS x 32 KB
  uint8_t* k_tile = tiles + GROUPS * TILE_BYTES;      // 2 x 32 KB
  uint8_t* v_tile = k_tile + 2 * TILE_BYTES;          // 2 x 32 KB
  TcSmem* sh = reinterpret_cast<TcSmem*>(v_tile + 2 * TILE_BYTES);
  constexpr bool CAPPED = FORM != FORM_PLAIN, BIASED = FORM == FORM_BIASED;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // one-dimensional grid, query tile slowest: every head's late tiles (most keys) are handed out before any early
  // tile, so the long CTAs start first on all SMs and the short ones fill the tail
  const int hq = (int)(blockIdx.x % (unsigned)p.hq);
  const int h = hq / (p.hq / p.hkv);

  // (sequence, query tile of 256 rows) of this CTA: late tiles (most keys) first
  int b = 0, tile_in_seq = 0;
  {
    int rem = (int)(gridDim.x / (unsigned)p.hq) - 1 - (int)(blockIdx.x / (unsigned)p.hq);
    for (; b < p.num_seqs; ++b) {
      const int n = p.q_indptr[b + 1] - p.q_indptr[b];
      const int nt = (n + BQ2 - 1) / BQ2;
      if (rem < nt) {
        tile_in_seq = rem;
        break;
      }
      rem -= nt;
    }
    if (b >= p.num_seqs) return;
  }
  if (threadIdx.x == 0) {
    mbar_init(&sh->q_full, 1);
    for (int s2 = 0; s2 < 2; ++s2) {
      mbar_init(&sh->k_full[s2], 1);
      mbar_init(&sh->k_empty[s2], 1);
      mbar_init(&sh->v_full[s2], 1);
      mbar_init(&sh->v_empty[s2], 1);
    }
    for (int g = 0; g < GROUPS; ++g) {
      mbar_init(&sh->s_full[g], 1);
      mbar_init(&sh->p_ready[g], 4);
      mbar_init(&sh->o_full[g], 1);
    }
    sh->abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_kv);
  }
  if (warp == 1) {
    tmem_alloc(&sh->tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sh->tmem_slot;  // columns: S of group g at 128 g (P overwrites its first 64), O of group g at 256 + 128 g
  volatile int* abort_flag = &sh->abort_flag;
  PG_PDL_ENTRY();

  const int q0 = p.q_indptr[b], q_len = p.q_indptr[b + 1] - q0;
  const int kv_len = p.kv_lens[b];
  const int row_base = tile_in_seq * BQ2;
  const int rows_here = min(BQ2, q_len - row_base);
  const int pos_base = kv_len - q_len + row_base;  // position of the CTA's first row
  const int j0 = BIASED && p.window > 0 ? max(0, pos_base - p.window + 1) / BKV : 0;
  // tiles of 128 keys each group needs: up to its last row's position
  int n_g[GROUPS];
#pragma unroll
  for (int g = 0; g < GROUPS; ++g) {
    const int rows_of_g = min(128, rows_here - g * 128);
    n_g[g] = (rows_of_g > 0 && kv_len > 0) ? min(pos_base + g * 128 + rows_of_g - 1, kv_len - 1) / BKV + 1 - j0 : 0;
  }
  const int n_tiles = max(n_g[0], n_g[1]);
  const int* table_row = p.table + (long long)b * p.table_stride;

  if (warp == 0) {
    // Producer warp.  A key tile and its value tile arrive as 4 * ppt small boxes (one per page, 64-column half and
    // K or V); the lanes issue them side by side, slot = lane, lane + 32, and each lane reads the page ids of its own
    // slots one tile ahead, so that neither the table's memory latency nor a serial run of TMA issues sits between
    // two tiles.
    if (n_tiles > 0) {
      const uint64_t pol = l2_policy_evict_normal();
      if (lane == 0) {
        mbar_expect_tx(&sh->q_full, GROUPS * TILE_BYTES);
#pragma unroll
        for (int g = 0; g < GROUPS; ++g) {
          tma_load_3d(q_tile + g * TILE_BYTES, &tm_q, &sh->q_full, 0, hq, q0 + row_base + g * 128, pol);
          tma_load_3d(q_tile + g * TILE_BYTES + HALF_BYTES, &tm_q, &sh->q_full, 64, hq, q0 + row_base + g * 128, pol);
        }
      }
      const int ppt = BKV / p.page_size;  // pages per key tile (1 .. 16)
      const int per_kv = 2 * ppt, slots = 4 * ppt;
      auto page_of = [&](int j, int slot) -> int {
        const int pg = (slot % per_kv) >> 1;
        const int pages_live = min(ppt, (kv_len - (j0 + j) * BKV + p.page_size - 1) / p.page_size);
        int page = (slot < slots && pg < pages_live) ? __ldg(table_row + (j0 + j) * ppt + pg) : 0;  // past the end: the padding page, keys masked
        if (page < 0 || page >= p.num_pages) {
          atomicCAS(p.status, PG_ST_OK, PG_ST_BOUNDS | (41u << 8));
          page = 0;
        }
        return page;
      };
      int nxt0 = page_of(0, lane), nxt1 = page_of(0, lane + 32);
      bool ok = true;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int pg0 = nxt0, pg1 = nxt1;
        if (j + 1 < n_tiles) {
          nxt0 = page_of(j + 1, lane);
          nxt1 = page_of(j + 1, lane + 32);
        }
        const int st = j & 1;
        if (j >= 2) {
          const uint32_t par = (uint32_t)(((j >> 1) - 1) & 1);
          ok = mbar_wait(&sh->k_empty[st], par, abort_flag) && mbar_wait(&sh->v_empty[st], par, abort_flag);
          ok = __all_sync(0xFFFFFFFFu, ok);
          if (!ok) break;
        }
        if (lane == 0) {
          mbar_expect_tx(&sh->k_full[st], TILE_BYTES);
          mbar_expect_tx(&sh->v_full[st], TILE_BYTES);
        }
        __syncwarp();
#pragma unroll
        for (int it = 0; it < 2; ++it) {
          const int slot = lane + 32 * it;
          if (slot < slots) {
            const int kvsel = slot / per_kv, rem = slot % per_kv, pg = rem >> 1, half = rem & 1;
            const int z = ((it ? pg1 : pg0) * 2 + kvsel) * p.page_size;
            uint8_t* dst = (kvsel ? v_tile : k_tile) + st * TILE_BYTES + half * HALF_BYTES + pg * p.page_size * 128;
            tma_load_3d(dst, &tm_kv, kvsel ? &sh->v_full[st] : &sh->k_full[st], half * 64, h, z, pol);
          }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && n_tiles > 0) {
      constexpr uint32_t idesc_s = idesc_bf16(128, 128, 0);
      constexpr uint32_t idesc_o = idesc_bf16(128, 128, 1);
      const uint32_t lbo = p.mn_lbo_first ? (uint32_t)HALF_BYTES : 1024u, sbo = p.mn_lbo_first ? 1024u : (uint32_t)HALF_BYTES;
      bool ok = mbar_wait(&sh->q_full, 0, abort_flag);
      int k_seen = -1, v_seen = -1;  // tiles whose K / V arrival this thread has already observed
      // S of group g, tile j.  K_j is released once the last group that needs it has issued its S.  S of tile j
      // overwrites the group's previous S and P: the tensor core runs this thread's instructions in order, and the
      // product that read that P was issued before.
      auto issue_s = [&](int g, int j) {
        if (j >= n_g[g]) return true;
        const int st = j & 1;
        if (k_seen < j) {
          if (!mbar_wait(&sh->k_full[st], (uint32_t)((j >> 1) & 1), abort_flag)) return false;
          k_seen = j;
        }
        tc_fence_after();
        const uint32_t qa = smem_u32(q_tile + g * TILE_BYTES), ka = smem_u32(k_tile + st * TILE_BYTES);
#pragma unroll
        for (int kb = 0; kb < 2; ++kb)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ss(tmem + (uint32_t)(g * 128), umma_desc_k_sw128(qa + kb * HALF_BYTES + k * 32), umma_desc_k_sw128(ka + kb * HALF_BYTES + k * 32), idesc_s,
                         (kb | k) ? 1u : 0u);
        umma_commit(&sh->s_full[g]);
        const bool last_user = (g == GROUPS - 1) || j >= n_g[GROUPS - 1];
        if (last_user) umma_commit(&sh->k_empty[st]);
        return true;
      };
      // O_g (+)= P_g V_j with P_g read from tensor memory.  V_j is released once the last group that needs it has
      // issued its product.
      auto issue_pv = [&](int g, int j) {
        if (j >= n_g[g]) return true;
        const int st = j & 1;
        if (!mbar_wait(&sh->p_ready[g], (uint32_t)(j & 1), abort_flag)) return false;
        if (v_seen < j) {
          if (!mbar_wait(&sh->v_full[st], (uint32_t)((j >> 1) & 1), abort_flag)) return false;
          v_seen = j;
        }
        tc_fence_after();
        const uint32_t va = smem_u32(v_tile + st * TILE_BYTES);
#pragma unroll
        for (int ks = 0; ks < 8; ++ks)
          umma_bf16_ts(tmem + 256u + (uint32_t)(g * 128), tmem + (uint32_t)(g * 128) + (uint32_t)(ks * 8), umma_desc_mn_sw128(va + ks * 2048, lbo, sbo), idesc_o,
                       (j | ks) ? 1u : 0u);
        umma_commit(&sh->o_full[g]);
        const bool last_user = (g == GROUPS - 1) || j >= n_g[GROUPS - 1];
        if (last_user) umma_commit(&sh->v_empty[st]);
        return true;
      };
      ok = ok && issue_s(0, 0) && issue_s(1, 0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        // while one group's softmax runs, the tensor core has the other group's product and next scores to do
        ok = issue_pv(0, j) && issue_s(0, j + 1) && issue_pv(1, j) && issue_s(1, j + 1);
      }
    }
  } else {
    // softmax / output warps: group g = one query tile, one row per thread (TMEM lane 32 * (warp % 4) + lane)
    const int g = (warp - 2) >> 2, wq = warp & 3;
    const int r = wq * 32 + lane;
    const int my_n = n_g[g];
    const int pos0 = pos_base + g * 128;  // position of the group's first row
    const int my_pos = pos0 + r;          // rows past the sequence compute garbage that is never stored
    const uint32_t s_row = tmem + ((uint32_t)(wq * 32) << 16) + (uint32_t)(g * 128);
    const uint32_t o_row = s_row + 256u;
    float m = -INFINITY, l = 0.f;  // m: the maximum the exponentials refer to (may lag the true maximum by up to 2^8)
    // bias per position in units of the raw (or capped) score, which scale_log2 turns into log2
    const float slope = BIASED && p.slopes ? p.slopes[hq] * 1.4426950408889634f / p.scale_log2 : 0.f;
    bool ok = true;
    // One key tile of this group.  MASK (a tile that the causal edge or the end of the keys crosses) is a compile-time
    // property: the plain tiles, nearly all of them, carry no compare or select per element.
    auto tile = [&](int j, auto mask_tag) -> bool {
      constexpr bool MASK = decltype(mask_tag)::value;
      if (!mbar_wait(&sh->s_full[g], (uint32_t)(j & 1), abort_flag)) return false;
      tc_fence_after();
      const int key0 = (j0 + j) * BKV;
      const int limit = min(my_pos, kv_len - 1) - key0;                                      // columns lo + 1 .. limit are visible to this row
      const int lo = BIASED && p.window > 0 ? my_pos - p.window - key0 : -1;
      // the whole row of S goes to registers in one round trip (four loads in flight, one wait): both the maximum
      // and the exponentials work from there, and S in tensor memory may be overwritten by P right away
      uint32_t v[BKV];
      tmem_ld32(s_row, v);
      tmem_ld32(s_row + 32, v + 32);
      tmem_ld32(s_row + 64, v + 64);
      tmem_ld32(s_row + 96, v + 96);
      tmem_ld_wait();
      if constexpr (CAPPED) {
        if (p.cap_in > 0.f) {
          float big = 0.f;
#pragma unroll
          for (int i = 0; i < BKV; i += 2) big = max3(big, fabsf(__uint_as_float(v[i])), fabsf(__uint_as_float(v[i + 1])));
          if (__any_sync(0xFFFFFFFFu, big * p.cap_in > 1.f)) {
#pragma unroll
            for (int i = 0; i < BKV; ++i) v[i] = __float_as_uint(tanh_ex2(__uint_as_float(v[i]) * p.cap_in));
          } else {
            const float2 ci = make_float2(p.cap_in, p.cap_in);
#pragma unroll
            for (int i = 0; i < BKV; i += 2) {
              const float2 t = tanh2_poly(__fmul2_rn(make_float2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), ci));
              v[i] = __float_as_uint(t.x);
              v[i + 1] = __float_as_uint(t.y);
            }
          }
        }
      }
      if constexpr (BIASED) {
        const float2 away = make_float2((float)(key0 - my_pos), (float)(key0 - my_pos)), sl = make_float2(slope, slope);
#pragma unroll
        for (int i = 0; i < BKV; i += 2) {
          const float2 t = __ffma2_rn(__fadd2_rn(make_float2((float)i, (float)(i + 1)), away), sl, make_float2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])));
          v[i] = __float_as_uint(t.x);
          v[i + 1] = __float_as_uint(t.y);
        }
      }
      float mx_raw;
      if constexpr (MASK) {
        mx_raw = -INFINITY;
#pragma unroll
        for (int i = 0; i < BKV; ++i)
          if (i <= limit && (!BIASED || i > lo)) mx_raw = fmaxf(mx_raw, __uint_as_float(v[i]));
      } else {
        // three-input maximum, four chains instead of one long one
        float m0 = max3(__uint_as_float(v[0]), __uint_as_float(v[1]), __uint_as_float(v[2]));
        float m1 = max3(__uint_as_float(v[3]), __uint_as_float(v[4]), __uint_as_float(v[5]));
        float m2 = max3(__uint_as_float(v[6]), __uint_as_float(v[7]), __uint_as_float(v[8]));
        float m3 = max3(__uint_as_float(v[9]), __uint_as_float(v[10]), __uint_as_float(v[11]));
#pragma unroll
        for (int i = 12; i + 7 < BKV; i += 8) {
          m0 = max3(m0, __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
          m1 = max3(m1, __uint_as_float(v[i + 2]), __uint_as_float(v[i + 3]));
          m2 = max3(m2, __uint_as_float(v[i + 4]), __uint_as_float(v[i + 5]));
          m3 = max3(m3, __uint_as_float(v[i + 6]), __uint_as_float(v[i + 7]));
        }
        // 12 + 8 * 14 = 124: four columns left
        m0 = max3(m0, __uint_as_float(v[124]), __uint_as_float(v[125]));
        m1 = max3(m1, __uint_as_float(v[126]), __uint_as_float(v[127]));
        mx_raw = fmaxf(max3(m0, m1, m2), m3);
      }
      const float mx = mx_raw * p.scale_log2;
      // the previous product of this group must be complete before O is rescaled
      if (j >= 1) {
        if (!mbar_wait(&sh->o_full[g], (uint32_t)((j - 1) & 1), abort_flag)) return false;
        tc_fence_after();
      }
      // move to a new maximum only when it grew by more than the threshold (or there was none yet)
      float alpha = 1.f;
      if (mx > m + RESCALE_LOG2 || (m == -INFINITY && mx > -INFINITY)) {
        alpha = (m == -INFINITY) ? 0.f : ex2_approx(m - mx);
        m = mx;
      }
      if (j >= 1 && __any_sync(0xFFFFFFFFu, alpha != 1.f)) {
        const float2 a2 = make_float2(alpha, alpha);
#pragma unroll 1
        for (int c = 0; c < D; c += 32) {
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
      // P = exp2(S * scale - m) as bf16, two per 32-bit column, over the first 64 columns of S; row sum
      float2 sum2 = make_float2(0.f, 0.f), sum3 = make_float2(0.f, 0.f);
      const float2 sc2 = make_float2(p.scale_log2, p.scale_log2), ng2 = make_float2(neg, neg);
#pragma unroll
      for (int c = 0; c < BKV; c += 32) {
        uint32_t packed[16];
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          const float2 t2 = __ffma2_rn(make_float2(__uint_as_float(v[c + i]), __uint_as_float(v[c + i + 1])), sc2, ng2);
          const float2 t3 = __ffma2_rn(make_float2(__uint_as_float(v[c + i + 2]), __uint_as_float(v[c + i + 3])), sc2, ng2);
          float2 e = make_float2(ex2_approx(t2.x), ex2_approx(t2.y));
          float2 f = make_float2(ex2_approx(t3.x), ex2_approx(t3.y));
          if constexpr (MASK) {
            if (c + i > limit || (BIASED && c + i <= lo)) e.x = 0.f;
            if (c + i + 1 > limit || (BIASED && c + i + 1 <= lo)) e.y = 0.f;
            if (c + i + 2 > limit || (BIASED && c + i + 2 <= lo)) f.x = 0.f;
            if (c + i + 3 > limit || (BIASED && c + i + 3 <= lo)) f.y = 0.f;
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
      if (lane == 0) mbar_arrive(&sh->p_ready[g]);
      return true;
    };
    for (int j = 0; j < my_n && ok; ++j) {
      const int key0 = (j0 + j) * BKV;
      const bool need_mask = key0 + BKV - 1 > min(pos0, kv_len - 1) || (BIASED && p.window > 0 && key0 <= pos0 + 127 - p.window);
      ok = need_mask ? tile(j, std::true_type{}) : tile(j, std::false_type{});
    }
    const int rows_g = min(128, rows_here - g * 128);
    if (ok && my_n > 0) {
      ok = mbar_wait(&sh->o_full[g], (uint32_t)((my_n - 1) & 1), abort_flag);
      tc_fence_after();
    }
    float inv = (ok && l > 0.f) ? 1.f / l : 0.f;
    if constexpr (CAPPED) {
      inv *= p.out_scale;
      if (p.gate && r < rows_g) inv /= 1.f + __expf(-__bfloat162float(p.gate[(long long)(q0 + row_base + g * 128 + r) * p.ld_gate + hq]));
    }
    bf16* dst = p.out + (CAPPED ? (q0 + row_base + g * 128 + r) * p.ld_out + hq * D : ((long long)(q0 + row_base + g * 128 + r) * p.hq + hq) * D);
#pragma unroll
    for (int c = 0; c < D; c += 32) {
      uint32_t w[32];
      if (my_n > 0) {  // uniform per group
        tmem_ld32(o_row + c, w);
        tmem_ld_wait();
      }
      if (r < rows_g) {
#pragma unroll
        for (int c8 = 0; c8 < 32; c8 += 8) {
          float f[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) f[i] = my_n > 0 ? __uint_as_float(w[c8 + i]) * inv : 0.f;
          *reinterpret_cast<bf16x8*>(dst + c + c8) = pack8(f);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
  if (threadIdx.x == 0 && sh->abort_flag) atomicCAS(p.status, PG_ST_OK, PG_ST_TIMEOUT | (41u << 8));
}


// ---------------------------------------------------------------------------------------------------------------------
// Head dim 256 (the gated full-attention layers of the hybrid models).  O of one 128-row query tile already takes 256 of
// the 512 TMEM columns, so a CTA owns ONE query tile and keeps the tensor core busy the other way round: the scores are
// double-buffered (tiles of 64 keys, S_j at columns 256 + 64 (j & 1)), and the MMA thread issues  P V of tile j, then S of
// tile j + 2  while the softmax warps work on tile j + 1.  Shared memory: Q 64 KB, K and V two stages of 32 KB each.
// The producer warp is split: lanes 0-15 feed K, lanes 16-31 feed V, each half with its own waits, because K runs two
// tiles ahead of V.
constexpr int D2 = 256, BQ1 = 128;
constexpr int Q2_BYTES = BQ1 * D2 * 2;     // 64 KB: [4 blocks of 64 columns][128 rows][128 B]
constexpr int KV2_BYTES = BKV2 * D2 * 2;   // 32 KB: [4 blocks of 64 columns][64 rows][128 B]
constexpr int KV2_BLOCK = BKV2 * 128;      // 8 KB
constexpr int THREADS2 = 64 + 128;

struct TcSmem2 {
  uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2], p_ready[2], o_full;
  uint32_t tmem_slot;
  int abort_flag;
};

__global__ void __launch_bounds__(THREADS2, 1) prefill_attn_tc256_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv, const TcAttnParams p) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = smem_u32(smem_raw);
  uint8_t* tiles = smem_raw + (((base + 1023u) & ~1023u) - base);
  uint8_t* q_tile = tiles;
  uint8_t* k_tile = tiles + Q2_BYTES;
  uint8_t* v_tile = k_tile + 2 * KV2_BYTES;
  TcSmem2* sh = reinterpret_cast<TcSmem2*>(v_tile + 2 * KV2_BYTES);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hq = (int)(blockIdx.x % (unsigned)p.hq);
  const int h = hq / (p.hq / p.hkv);
  int b = 0, tile_in_seq = 0;  // late tiles (most keys) first, every head's before any early tile
  {
    int rem = (int)(gridDim.x / (unsigned)p.hq) - 1 - (int)(blockIdx.x / (unsigned)p.hq);
    for (; b < p.num_seqs; ++b) {
      const int n = p.q_indptr[b + 1] - p.q_indptr[b];
      const int nt = (n + BQ1 - 1) / BQ1;
      if (rem < nt) {
        tile_in_seq = rem;
        break;
      }
      rem -= nt;
    }
    if (b >= p.num_seqs) return;
  }
  if (threadIdx.x == 0) {
    mbar_init(&sh->q_full, 1);
    for (int s2 = 0; s2 < 2; ++s2) {
      mbar_init(&sh->k_full[s2], 1);
      mbar_init(&sh->k_empty[s2], 1);
      mbar_init(&sh->v_full[s2], 1);
      mbar_init(&sh->v_empty[s2], 1);
      mbar_init(&sh->s_full[s2], 1);
      mbar_init(&sh->p_ready[s2], 4);
    }
    mbar_init(&sh->o_full, 1);
    sh->abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_kv);
  }
  if (warp == 1) {
    tmem_alloc(&sh->tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sh->tmem_slot;  // columns: O at 0 .. 255, S / P of tile j at 256 + 64 (j & 1)
  volatile int* abort_flag = &sh->abort_flag;
  PG_PDL_ENTRY();

  const int q0 = p.q_indptr[b], q_len = p.q_indptr[b + 1] - q0;
  const int kv_len = p.kv_lens[b];
  const int row_base = tile_in_seq * BQ1;
  const int rows_here = min(BQ1, q_len - row_base);
  const int pos0 = kv_len - q_len + row_base;  // position of the tile's first row
  // key tiles j0 .. last the rows of this tile can see (a sliding window drops the tiles in front of the first row's
  // window); the loops below count tiles from j0
  const int j0 = (p.window > 0 && rows_here > 0) ? max(0, pos0 - p.window + 1) / BKV2 : 0;
  const int n_tiles = (rows_here > 0 && kv_len > 0) ? min(pos0 + rows_here - 1, kv_len - 1) / BKV2 + 1 - j0 : 0;
  const int* table_row = p.table + (long long)b * p.table_stride;

  if (warp == 0) {
    if (n_tiles > 0) {
      const uint64_t pol = l2_policy_evict_normal();
      if (lane == 0) {
        mbar_expect_tx(&sh->q_full, Q2_BYTES);
#pragma unroll
        for (int cb = 0; cb < 4; ++cb) tma_load_3d(q_tile + cb * (BQ1 * 128), &tm_q, &sh->q_full, cb * 64, hq, q0 + row_base, pol);
      }
      // lanes 0-15: K boxes, lanes 16-31: V boxes; slot = (page of the tile, 64-column block), 4 * ppt slots per tile
      const int kvsel = lane >> 4, sub = lane & 15;
      const uint32_t half_mask = kvsel ? 0xFFFF0000u : 0x0000FFFFu;
      const int ppt = BKV2 / p.page_size;  // 1 .. 8
      const int slots = 4 * ppt;           // 4 .. 32: up to two per lane
      uint64_t* full = kvsel ? sh->v_full : sh->k_full;
      uint64_t* empty = kvsel ? sh->v_empty : sh->k_empty;
      uint8_t* tile0 = kvsel ? v_tile : k_tile;
      auto page_of = [&](int j, int slot) -> int {
        const int pg = slot >> 2;
        const int pages_live = min(ppt, (kv_len - j * BKV2 + p.page_size - 1) / p.page_size);
        int page = (slot < slots && pg < pages_live) ? __ldg(table_row + j * ppt + pg) : 0;  // past the end: the padding page, keys masked
        if (page < 0 || page >= p.num_pages) {
          atomicCAS(p.status, PG_ST_OK, PG_ST_BOUNDS | (42u << 8));
          page = 0;
        }
        return page;
      };
      int nxt0 = page_of(j0, sub), nxt1 = page_of(j0, sub + 16);
      for (int j = 0; j < n_tiles; ++j) {
        const int pg0 = nxt0, pg1 = nxt1;
        if (j + 1 < n_tiles) {
          nxt0 = page_of(j0 + j + 1, sub);
          nxt1 = page_of(j0 + j + 1, sub + 16);
        }
        const int st = j & 1;
        if (j >= 2) {
          bool ok = mbar_wait(&empty[st], (uint32_t)(((j >> 1) - 1) & 1), abort_flag);
          ok = __all_sync(half_mask, ok);
          if (!ok) break;
        }
        if (sub == 0) mbar_expect_tx(&full[st], KV2_BYTES);
        __syncwarp(half_mask);
#pragma unroll
        for (int it = 0; it < 2; ++it) {
          const int slot = sub + 16 * it;
          if (slot < slots) {
            const int pg = slot >> 2, cb = slot & 3;
            const int z = ((it ? pg1 : pg0) * 2 + kvsel) * p.page_size;
            tma_load_3d(tile0 + st * KV2_BYTES + cb * KV2_BLOCK + pg * p.page_size * 128, &tm_kv, &full[st], cb * 64, h, z, pol);
          }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && n_tiles > 0) {
      constexpr uint32_t idesc_s = idesc_bf16(128, BKV2, 0);
      constexpr uint32_t idesc_o = idesc_bf16(128, D2, 1);
      const uint32_t lbo = p.mn_lbo_first ? (uint32_t)KV2_BLOCK : 1024u, sbo = p.mn_lbo_first ? 1024u : (uint32_t)KV2_BLOCK;
      bool ok = mbar_wait(&sh->q_full, 0, abort_flag);
      // S of tile j into buffer j & 1.  It overwrites S and P of tile j - 2: the product that read that P was issued
      // before, and the tensor core runs this thread's instructions in order.
      auto issue_s = [&](int j) {
        if (j >= n_tiles) return true;
        const int st = j & 1;
        if (!mbar_wait(&sh->k_full[st], (uint32_t)((j >> 1) & 1), abort_flag)) return false;
        tc_fence_after();
        const uint32_t qa = smem_u32(q_tile), ka = smem_u32(k_tile + st * KV2_BYTES);
#pragma unroll
        for (int cb = 0; cb < 4; ++cb)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ss(tmem + 256u + (uint32_t)(st * BKV2), umma_desc_k_sw128(qa + cb * (BQ1 * 128) + k * 32), umma_desc_k_sw128(ka + cb * KV2_BLOCK + k * 32), idesc_s,
                         (cb | k) ? 1u : 0u);
        umma_commit(&sh->s_full[st]);
        umma_commit(&sh->k_empty[st]);
        return true;
      };
      ok = ok && issue_s(0) && issue_s(1);
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int st = j & 1;
        ok = mbar_wait(&sh->p_ready[st], (uint32_t)((j >> 1) & 1), abort_flag) && mbar_wait(&sh->v_full[st], (uint32_t)((j >> 1) & 1), abort_flag);
        if (!ok) break;
        tc_fence_after();
        const uint32_t va = smem_u32(v_tile + st * KV2_BYTES);
#pragma unroll
        for (int ks = 0; ks < BKV2 / 16; ++ks)
          umma_bf16_ts(tmem, tmem + 256u + (uint32_t)(st * BKV2) + (uint32_t)(ks * 8), umma_desc_mn_sw128(va + ks * 2048, lbo, sbo), idesc_o, (j | ks) ? 1u : 0u);
        umma_commit(&sh->o_full);
        umma_commit(&sh->v_empty[st]);
        ok = issue_s(j + 2);
      }
    }
  } else {
    // softmax / output warps: one query row per thread (TMEM lane 32 * (warp % 4) + lane)
    const int wq = warp & 3;
    const int r = wq * 32 + lane;
    const int my_pos = pos0 + r;  // rows past the sequence compute garbage that is never stored
    const uint32_t lane_base = tmem + ((uint32_t)(wq * 32) << 16);
    const uint32_t o_row = lane_base;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int key0 = (j0 + j) * BKV2;
      // a tile needs the mask when the causal edge or the end of the keys crosses it, or (sliding window) when its first
      // key lies in front of the window of the tile's last row
      const bool need_mask = key0 + BKV2 - 1 > min(pos0, kv_len - 1) || (p.window > 0 && key0 <= pos0 + BQ1 - 1 - p.window);
      const int st = j & 1;
      const uint32_t s_row = lane_base + 256u + (uint32_t)(st * BKV2);
      const int limit = min(my_pos, kv_len - 1) - key0;                          // columns lo + 1 .. limit are visible to this row
      const int lo = p.window > 0 ? my_pos - p.window - key0 : -(1 << 30);
      const uint32_t sp = (uint32_t)((j >> 1) & 1), op = (uint32_t)((j - 1) & 1);
      ok = need_mask ? softmax_tile64<true>(&sh->s_full[st], sp, s_row, o_row, D2, &sh->o_full, op, j, limit, lo, p.scale_log2, m, l, &sh->p_ready[st], lane, abort_flag)
                     : softmax_tile64<false>(&sh->s_full[st], sp, s_row, o_row, D2, &sh->o_full, op, j, limit, lo, p.scale_log2, m, l, &sh->p_ready[st], lane, abort_flag);
    }
    if (ok && n_tiles > 0) {
      ok = mbar_wait(&sh->o_full, (uint32_t)((n_tiles - 1) & 1), abort_flag);
      tc_fence_after();
    }
    const float inv = (ok && l > 0.f) ? 1.f / l : 0.f;
    bf16* dst = p.out + ((long long)(q0 + row_base + r) * p.hq + hq) * D2;
#pragma unroll 1
    for (int c = 0; c < D2; c += 32) {
      uint32_t w[32];
      if (n_tiles > 0) {
        tmem_ld32(o_row + c, w);
        tmem_ld_wait();
      }
      if (r < rows_here) {
#pragma unroll
        for (int c8 = 0; c8 < 32; c8 += 8) {
          float f[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) f[i] = n_tiles > 0 ? __uint_as_float(w[c8 + i]) * inv : 0.f;
          *reinterpret_cast<bf16x8*>(dst + c + c8) = pack8(f);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
  if (threadIdx.x == 0 && sh->abort_flag) atomicCAS(p.status, PG_ST_OK, PG_ST_TIMEOUT | (42u << 8));
}


int g_mn_variant = -1;

}  // namespace

// Test hook: which of the two stride fields of the MN-major descriptor carries the 64-column block stride.
extern "C" void pg_prefill_attention_tc_variant(int v) { g_mn_variant = v; }

// q [T, hq, d] bf16 (contiguous), kv_layer [pages, 2, page_size, hkv, d], out [T, hq * d], d = 128 or 256.  `q_tiles` = sum
// over the sequences of ceil(query rows / 256) for d = 128 and of ceil(query rows / 128) for d = 256.
static int prefill_tc_impl(const void* q, const void* kv_layer, void* out, const void* q_indptr, const void* kv_lens, const void* table, int table_stride, int num_seqs, int tokens, int hq,
                           int hkv, int dim, int page_size, long long num_pages, float scale, int q_tiles, int window, int form, float softcap, const void* gate, long long ld_gate,
                           const void* slopes, float out_scale, long long ld_out, void* status, cudaStream_t stream);

extern "C" int pg_prefill_attention_tc(const void* q, const void* kv_layer, void* out, const void* q_indptr, const void* kv_lens, const void* table, int table_stride,
                                       int num_seqs, int tokens, int hq, int hkv, int dim, int page_size, long long num_pages, float scale, int q_tiles, int window,
                                       void* status, cudaStream_t stream) {
  return prefill_tc_impl(q, kv_layer, out, q_indptr, kv_lens, table, table_stride, num_seqs, tokens, hq, hkv, dim, page_size, num_pages, scale, q_tiles, window, FORM_PLAIN, 0.f, nullptr, 0,
                         nullptr, 1.f, (long long)hq * dim, status, stream);
}

// Head dim 128 with a soft cap on the scores (softcap > 0), a sigmoid gate per (token, head) (gate: bf16 rows or null), a sliding window
// (> 0), a bias of slope * distance (slopes: f32 [hq] or null); output rows of stride ld_out, times out_scale.
extern "C" int pg_prefill_attention_tc_capped(const void* q, const void* kv_layer, void* out, const void* q_indptr, const void* kv_lens, const void* table, int table_stride, int num_seqs,
                                              int tokens, int hq, int hkv, int page_size, long long num_pages, float scale, float softcap, const void* gate, long long ld_gate, int window,
                                              const void* slopes, float out_scale, long long ld_out, int q_tiles, void* status, cudaStream_t stream) {
  PG_REQUIRE(window >= 0 && ld_out % 8 == 0 && ((uintptr_t)out & 15) == 0, "tcgen05 prefill attention: a window of %d keys, output rows of %lld that must start on 16 bytes", window, ld_out);
  return prefill_tc_impl(q, kv_layer, out, q_indptr, kv_lens, table, table_stride, num_seqs, tokens, hq, hkv, D, page_size, num_pages, scale, q_tiles, window,
                         window > 0 || slopes ? FORM_BIASED : FORM_CAPPED, softcap, gate, ld_gate, slopes, out_scale, ld_out, status, stream);
}

static int prefill_tc_impl(const void* q, const void* kv_layer, void* out, const void* q_indptr, const void* kv_lens, const void* table, int table_stride, int num_seqs, int tokens, int hq,
                           int hkv, int dim, int page_size, long long num_pages, float scale, int q_tiles, int window, int form, float softcap, const void* gate, long long ld_gate,
                           const void* slopes, float out_scale, long long ld_out, void* status, cudaStream_t stream) {
  PG_REQUIRE(window == 0 || dim == D2 || form == FORM_BIASED, "tcgen05 prefill attention: a sliding window is built for head dim 256 and the biased form only");
  PG_REQUIRE(dim == D || dim == D2, "tcgen05 prefill attention is built for head dims 128 and 256 (got %d)", dim);
  const int key_tile = dim == D ? BKV : BKV2;
  PG_REQUIRE(page_size >= 8 && page_size <= key_tile && key_tile % page_size == 0, "page size %d does not tile %d keys", page_size, key_tile);
  PG_REQUIRE(num_pages * 2 * page_size < (1ll << 31), "KV cache of %lld pages is too large for 32-bit TMA row coordinates", num_pages);
  PG_REQUIRE(hq % hkv == 0, "query heads %d are not a multiple of the KV heads %d", hq, hkv);
  if (q_tiles == 0 || tokens == 0) return PG_OK;
  CUtensorMap tm_q, tm_kv;
  int rc = make_tmap_rows_heads(&tm_q, q, tokens, hq, 128, dim);
  if (rc != PG_OK) return rc;
  rc = make_tmap_rows_heads(&tm_kv, kv_layer, num_pages * 2 * page_size, hkv, page_size, dim);
  if (rc != PG_OK) return rc;
  TcAttnParams p;
  p.out = (bf16*)out;
  p.q_indptr = (const int*)q_indptr;
  p.kv_lens = (const int*)kv_lens;
  p.table = (const int*)table;
  p.table_stride = table_stride;
  p.num_seqs = num_seqs;
  p.hq = hq;
  p.hkv = hkv;
  p.page_size = page_size;
  p.num_pages = num_pages;
  p.scale_log2 = (softcap > 0.f ? softcap : scale) * 1.4426950408889634f;
  p.cap_in = softcap > 0.f ? scale / softcap : 0.f;
  p.gate = (const bf16*)gate;
  p.ld_gate = ld_gate;
  p.window = window;
  p.slopes = (const float*)slopes;
  p.out_scale = out_scale;
  p.ld_out = ld_out;
  p.mn_lbo_first = g_mn_variant < 0 ? 1 : g_mn_variant;
  p.status = (uint32_t*)status;
  if (dim == D2) {
    const size_t smem2 = 1024 + (size_t)Q2_BYTES + 4 * (size_t)KV2_BYTES + sizeof(TcSmem2) + 64;
    static bool attr2_done = false;
    if (!attr2_done) {
      PG_CUDA(cudaFuncSetAttribute(prefill_attn_tc256_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem2));
      attr2_done = true;
    }
    PG_CUDA(launch_pdl(prefill_attn_tc256_kernel, dim3((unsigned)q_tiles * (unsigned)hq), dim3(THREADS2), smem2, stream, tm_q, tm_kv, p));
    PG_LAUNCH_CHECK();
    return PG_OK;
  }
  const size_t smem = 1024 + (GROUPS + 4) * (size_t)TILE_BYTES + sizeof(TcSmem) + 64;
  static bool attr_done = false;
  if (!attr_done) {
    PG_CUDA(cudaFuncSetAttribute(prefill_attn_tc_kernel<FORM_PLAIN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    PG_CUDA(cudaFuncSetAttribute(prefill_attn_tc_kernel<FORM_CAPPED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    PG_CUDA(cudaFuncSetAttribute(prefill_attn_tc_kernel<FORM_BIASED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr_done = true;
  }
  PG_CUDA(launch_pdl(form == FORM_BIASED ? prefill_attn_tc_kernel<FORM_BIASED> : form == FORM_CAPPED ? prefill_attn_tc_kernel<FORM_CAPPED> : prefill_attn_tc_kernel<FORM_PLAIN>, dim3((unsigned)q_tiles * (unsigned)hq), dim3(THREADS), smem, stream, tm_q, tm_kv, p));
  PG_LAUNCH_CHECK();
  return PG_OK;
}

