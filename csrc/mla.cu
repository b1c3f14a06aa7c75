// Multi-head latent attention kernels (DeepSeek-V2-Lite / Kimi-K2 shapes).
//
//  * mla_append: RMSNorm of the compressed KV row, RoPE of the shared rope key
//    (interleaved-pair input -> half-split output), append [ckv | k_pe] to the paged
//    latent cache [pages, page_size, kv_lora + rope].
//  * mla_q_prep: RoPE on the query rope tail and a head-major copy of q_nope, so the
//    absorb step (q_nope * W_UK per head) can run on the grouped tcgen05 GEMM.
//  * mla_attn: absorbed attention over the latent cache.  All heads share one KV row per
//    token, so a CTA takes 16 heads of one query token as the 16 MMA rows and streams
//    32-token latent tiles (cp.async, double buffered).  The score contraction (576 wide at
//    512 + 64) is split over the four warps and summed through shared memory; each warp then
//    owns a quarter of the value dims for P*V.  Split-KV + merge for decode.  Instances for
//    latents up to 128, 256 and 512 with no or up to 64 rotated columns; smaller sizes
//    (multiples of 8) fill the rest of the tile with zeros in shared memory only.  A sliding
//    window skips the tiles in front of it.  Queries either come rotated, or their rotary part
//    is turned by f32 tables on its way into the MMA fragments (pairs of neighbouring columns).
//    A sink per head adds exp(sink) to the softmax's denominator, and the sigmoid of a gate per
//    (token, head) may multiply the output: both where a row is divided by its sum (or merged).
//  * latent_rows: from one token's fused projection row, the RMS-normed query latent (dense; none
//    where queries have no latent) and
//    the cache row: RMS-normed latent, then the shared key part rotated in pairs with f32 tables.
//    rotate_pairs_: the same rotation in place on the query columns, for the expanded prefill form.
//  * latent_attention_plain: the absorbed form on the CUDA cores for f32 and for sizes the tensor-core
//    kernel does not address.
//  * permute_021: [A, B, D] -> [B, A, D] row permutation (head-major <-> token-major).
//
// Functional parity with pegainfer-kernels/csrc/kimi_k2/kimi_mla.cu:83-885 (split/norm,
// rope, paged append, absorbed batch decode), csrc/deepseek_v2_lite/dsv2_lite_attention.cu
// and csrc/k3/k3_mla_paged_attn.cu (block-table walk, zero output for empty rows).
#include <float.h>

#include "api.h"
#include "common.cuh"
#include "types.cuh"

namespace {

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(sz) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  bf162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

constexpr float NEG_BIG = -1e30f;
constexpr float LOG2E = 1.4426950408889634f;

// one warp per token
__global__ void __launch_bounds__(128) mla_append_kernel(const bf16* __restrict__ kv_a, long long ld, const bf16* __restrict__ norm_w,
                                                          const bf16* __restrict__ cos, const bf16* __restrict__ sin, const int* __restrict__ positions,
                                                          const int* __restrict__ slots, bf16* __restrict__ latent, int tokens, int c, int rope,
                                                          int max_pos, long long num_slots, float eps, uint32_t* status) {
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= tokens) return;
  const long long slot = slots[t];
  if (slot < 0 || slot >= num_slots) {
    if (lane == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (6u << 8));
    return;
  }
  int pos = positions[t];
  if (pos < 0 || pos >= max_pos) {
    if (lane == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (7u << 8));
    pos = pos < 0 ? 0 : max_pos - 1;
  }
  const bf16* src = kv_a + t * ld;
  bf16* dst = latent + slot * (c + rope);
  float ss = 0.f;
  for (int i = lane; i < c; i += 32) {
    const float v = __bfloat162float(src[i]);
    ss += v * v;
  }
  ss = warp_sum(ss);
  const float inv = rsqrtf(ss / (float)c + eps);
  for (int i = lane; i < c; i += 32) dst[i] = __float2bfloat16(__bfloat162float(src[i]) * inv * __bfloat162float(norm_w[i]));
  const int half = rope / 2;
  for (int i = lane; i < half; i += 32) {
    const float x1 = __bfloat162float(src[c + 2 * i]), x2 = __bfloat162float(src[c + 2 * i + 1]);
    const float cs = __bfloat162float(cos[(long long)pos * half + i]), sn = __bfloat162float(sin[(long long)pos * half + i]);
    dst[c + i] = __float2bfloat16(x1 * cs - x2 * sn);
    dst[c + half + i] = __float2bfloat16(x2 * cs + x1 * sn);
  }
}

// one warp per (token, head): q [T, H, nope + rope] -> q_nope_hm [H, T, nope], q_pe [T, H, rope] (rotated)
__global__ void __launch_bounds__(128) mla_q_prep_kernel(const bf16* __restrict__ q, const bf16* __restrict__ cos, const bf16* __restrict__ sin,
                                                          const int* __restrict__ positions, bf16* __restrict__ q_nope_hm, bf16* __restrict__ q_pe,
                                                          int tokens, int heads, int nope, int rope, int max_pos) {
  const long long unit = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= (long long)tokens * heads) return;
  const int t = (int)(unit / heads), h = (int)(unit % heads);
  const bf16* src = q + unit * (nope + rope);
  bf16* dn = q_nope_hm + ((long long)h * tokens + t) * nope;
  for (int i = lane; i < nope / 8; i += 32) reinterpret_cast<uint4*>(dn)[i] = reinterpret_cast<const uint4*>(src)[i];
  int pos = positions[t];
  pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
  const int half = rope / 2;
  bf16* dp = q_pe + unit * rope;
  for (int i = lane; i < half; i += 32) {
    const float x1 = __bfloat162float(src[nope + 2 * i]), x2 = __bfloat162float(src[nope + 2 * i + 1]);
    const float cs = __bfloat162float(cos[(long long)pos * half + i]), sn = __bfloat162float(sin[(long long)pos * half + i]);
    dp[i] = __float2bfloat16(x1 * cs - x2 * sn);
    dp[half + i] = __float2bfloat16(x2 * cs + x1 * sn);
  }
}

__global__ void permute_021_kernel(const bf16* __restrict__ in, bf16* __restrict__ out, int A, int B, int D) {
  const long long row = blockIdx.x;  // output row index b * A + a
  const int b = (int)(row / A), a = (int)(row % A);
  const uint4* src = reinterpret_cast<const uint4*>(in + ((long long)a * B + b) * D);
  uint4* dst = reinterpret_cast<uint4*>(out + row * D);
  for (int i = threadIdx.x; i < D / 8; i += blockDim.x) dst[i] = src[i];
}

struct MlaParams {
  const bf16* q_abs;   // [T, H, C] by strides
  const bf16* q_pe;    // [T, H, R] by strides
  const bf16* latent;  // [pages, ps, C + R]
  bf16* out;           // [T, H, C] by strides
  long long q_tok, q_head, pe_tok, pe_head, o_tok, o_head;
  const float* cos;    // [max_pos, R / 2]: rotate the query columns here (null: they come rotated)
  const float* sin;
  int max_pos;
  int c, r;            // sizes of the latent and the shared key part, at most the instance's
  int window;          // a row sees its last `window` keys (0: all of them)
  const int* q_indptr;
  const int* kv_lens;
  const int* table;
  int table_stride, num_seqs, tokens, heads, page_size, splits;
  float scale_log2;
  float* part_o;    // [tokens * heads, splits, C]
  float* part_lse;  // [tokens * heads, splits]
  const float* sink;    // [H]: exp(sink) is part of a row's denominator (null: none)
  const bf16* gate;     // [T, >= H] rows of stride ld_gate whose sigmoid multiplies a head's output (null: none)
  long long ld_gate;
  const int* unit_seq;  // [first_row + T] sequence of each token row
  int first_row;        // number of this launch's first row in the step
};

// Factor on a row's sum of weighted values: 1 / (sum of weights + sink), times the gate.  `m` and `l`: maximum (log2) and sum.
__device__ __forceinline__ float row_factor(const MlaParams& p, int t, int head, float m, float l) {
  if (!(l > 0.f)) return 0.f;
  if (p.sink) l += exp2f(p.sink[head] * LOG2E - m);
  float f = 1.f / l;
  if (p.gate) f /= 1.f + __expf(-__bfloat162float(p.gate[t * p.ld_gate + head]));
  return f;
}

// CTA = (token row t, head group of 16, split).  C, R: sizes of the instance; EXACT: they are the problem's.
template <int C, int R, bool EXACT>
__global__ void __launch_bounds__(128) mla_attn_kernel(const MlaParams p) {
  extern __shared__ __align__(128) uint8_t smem_raw[];
  constexpr int W = C + R;          // 576
  constexpr int TILE = 32;
  constexpr int CHUNKS = W / 8;     // 72 sixteen-byte chunks per row
  constexpr int KS_PER_WARP = (W / 16) / 4;  // 9
  constexpr int VD = C / 4;         // 128 value dims per warp
  constexpr int NT = VD / 8;        // 16
  static_assert(W % 64 == 0 && C % 64 == 0, "a row is split over four warps in steps of 16 columns");
  bf16* tile_sm = reinterpret_cast<bf16*>(smem_raw);                           // [2][TILE][W]
  float* s_part = reinterpret_cast<float*>(smem_raw + 2 * TILE * W * 2);     // [4 warps][16][TILE]
  PG_PDL_ENTRY();
  const int pc = EXACT ? C : p.c, pr = EXACT ? R : p.r;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, t4 = lane & 3;
  const int groups = (p.heads + 15) / 16;
  const int split = blockIdx.x % p.splits;
  const int hg = (blockIdx.x / p.splits) % groups;
  const int t = blockIdx.x / (p.splits * groups);
  const int b = p.unit_seq[p.first_row + t];
  const int q0 = p.q_indptr[b], q1 = p.q_indptr[b + 1];
  const int kv_len = p.kv_lens[b];
  const int pos = kv_len - (q1 - q0) + (p.first_row + t - q0);  // position of this query token
  const int kv_end = kv_len == 0 ? 0 : pos + 1;   // causal
  const int kv_begin = p.window > 0 ? max(0, kv_end - p.window) : 0;
  const int* table_row = p.table + (long long)b * p.table_stride;
  const int tile0 = kv_begin / TILE;
  const int n_tiles = (kv_end + TILE - 1) / TILE;
  const int tps = (n_tiles - tile0 + p.splits - 1) / p.splits;
  const int t_begin = tile0 + split * tps, t_end = min(n_tiles, t_begin + tps);

  auto swz = [](int r, int ch) { return r * W + ((ch ^ (r & 7)) << 3); };

  // Q fragments for this warp's slice of the columns of [q_abs | q_pe]
  uint32_t qf[KS_PER_WARP][4];
#pragma unroll
  for (int ks = 0; ks < KS_PER_WARP; ++ks) {
    const int d0 = (warp * KS_PER_WARP + ks) * 16;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
#pragma unroll
      for (int rr = 0; rr < 2; ++rr) {
        const int head = hg * 16 + g + rr * 8;
        const int d = d0 + half * 8 + 2 * t4;
        uint32_t v = 0u;
        if (head < p.heads) {
          if (d < C) {
            if (d < pc) v = *reinterpret_cast<const uint32_t*>(p.q_abs + t * p.q_tok + head * p.q_head + d);
          } else if (R > 0 && d - C < pr) {
            v = *reinterpret_cast<const uint32_t*>(p.q_pe + t * p.pe_tok + head * p.pe_head + (d - C));
            if (p.cos != nullptr) {
              const float2 f = __bfloat1622float2(*reinterpret_cast<const bf162*>(&v));
              const long long at = (long long)min(max(pos, 0), p.max_pos - 1) * (pr / 2) + (d - C) / 2;
              const float cs = p.cos[at], sn = p.sin[at];
              v = pack_bf16(f.x * cs - f.y * sn, f.y * cs + f.x * sn);
            }
          }
        }
        qf[ks][half * 2 + rr] = v;
      }
    }
  }
  float o[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m_run[2] = {NEG_BIG, NEG_BIG}, l_run[2] = {0.f, 0.f};

  // A 32-token tile starts at a multiple of 32 and pages hold 16, 32 or 64 tokens: at most two
  // page-table entries per tile, read once; a thread's 18 chunks follow by stepping (row, chunk)
  // instead of dividing by 72 and by the page size for every 16 bytes.
  const int ps_shift = __ffs(p.page_size) - 1;
  const int c0_r = threadIdx.x / CHUNKS, c0_ch = threadIdx.x % CHUNKS;
  auto issue = [&](int tile, int stage) {
    bf16* dst = tile_sm + stage * TILE * W;
    if (tile < t_end) {
      const int tok_base = tile * TILE;
      const int pf = tok_base >> ps_shift;
      const int pg0 = table_row[min(pf, p.table_stride - 1)];
      const int pg1 = (1 << ps_shift) < TILE ? table_row[min(pf + 1, p.table_stride - 1)] : pg0;
      int r = c0_r, ch = c0_ch;
#pragma unroll
      for (int i = 0; i < TILE * CHUNKS / 128; ++i) {
        const bool valid = tok_base + r < kv_end;
        const int rr = valid ? r : 0;
        const int page = (rr >> ps_shift) ? pg1 : pg0;
        // chunk `ch` of the tile row: latent columns, then (at C / 8) the rotated key part; the rest is zero
        const bool in_c = ch < C / 8;
        const int sch = in_c ? ch : ch - C / 8 + pc / 8;
        const bool live = valid && (in_c ? ch < pc / 8 : sch < (pc + pr) / 8);
        const bf16* src = p.latent + ((long long)page * p.page_size + ((tok_base + rr) & (p.page_size - 1))) * (pc + pr) + (live ? sch * 8 : 0);
        cp_async16(dst + swz(r, ch), src, live);
        ch += 128 % CHUNKS;
        r += 128 / CHUNKS;
        if (ch >= CHUNKS) {
          ch -= CHUNKS;
          ++r;
        }
      }
    }
    cp_async_commit();
  };

  issue(t_begin, 0);
  for (int tile = t_begin; tile < t_end; ++tile) {
    const int stage = (tile - t_begin) & 1;
    issue(tile + 1, stage ^ 1);
    cp_async_wait<1>();
    __syncthreads();
    const bf16* ts = tile_sm + stage * TILE * W;
    // partial scores over this warp's 144 dims: [16 heads x 32 tokens]
    float s_acc[TILE / 8][4];
#pragma unroll
    for (int n = 0; n < TILE / 8; ++n) s_acc[n][0] = s_acc[n][1] = s_acc[n][2] = s_acc[n][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < KS_PER_WARP; ++ks) {
      const int chb = (warp * KS_PER_WARP + ks) * 2;
#pragma unroll
      for (int n2 = 0; n2 < TILE / 16; ++n2) {
        const int j = lane >> 3, r = lane & 7;
        const int row = n2 * 16 + (j >> 1) * 8 + r;
        uint32_t b0, b1, b2, b3;
        ldsm_x4(smem_u32(ts + swz(row, chb + (j & 1))), b0, b1, b2, b3);
        mma16816(s_acc[2 * n2], qf[ks], b0, b1);
        mma16816(s_acc[2 * n2 + 1], qf[ks], b2, b3);
      }
    }
    float* mine = s_part + warp * 16 * TILE;
#pragma unroll
    for (int n = 0; n < TILE / 8; ++n) {
      mine[g * TILE + n * 8 + 2 * t4] = s_acc[n][0];
      mine[g * TILE + n * 8 + 2 * t4 + 1] = s_acc[n][1];
      mine[(g + 8) * TILE + n * 8 + 2 * t4] = s_acc[n][2];
      mine[(g + 8) * TILE + n * 8 + 2 * t4 + 1] = s_acc[n][3];
    }
    __syncthreads();
    float mx[2] = {NEG_BIG, NEG_BIG};
#pragma unroll
    for (int n = 0; n < TILE / 8; ++n) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = g + (e >> 1) * 8, col = n * 8 + 2 * t4 + (e & 1);
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) s += s_part[(w * 16 + row) * TILE + col];
        const int tok = tile * TILE + col;
        s = tok < kv_end && tok >= kv_begin ? s * p.scale_log2 : NEG_BIG;
        s_acc[n][e] = s;
        mx[e >> 1] = fmaxf(mx[e >> 1], s);
      }
    }
    float corr[2];
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 1));
      mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 2));
      const float m_new = fmaxf(m_run[rr], mx[rr]);
      corr[rr] = exp2f(m_run[rr] - m_new);
      m_run[rr] = m_new;
    }
    float ps[2] = {0.f, 0.f};
    uint32_t pa[TILE / 16][4];
#pragma unroll
    for (int n = 0; n < TILE / 8; ++n) {
      float pv[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        pv[e] = s_acc[n][e] <= NEG_BIG ? 0.f : exp2f(s_acc[n][e] - m_run[e >> 1]);
        ps[e >> 1] += pv[e];
      }
      pa[n >> 1][(n & 1) * 2 + 0] = pack_bf16(pv[0], pv[1]);
      pa[n >> 1][(n & 1) * 2 + 1] = pack_bf16(pv[2], pv[3]);
    }
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      ps[rr] += __shfl_xor_sync(0xffffffffu, ps[rr], 1);
      ps[rr] += __shfl_xor_sync(0xffffffffu, ps[rr], 2);
      l_run[rr] = l_run[rr] * corr[rr] + ps[rr];
    }
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      o[n][0] *= corr[0];
      o[n][1] *= corr[0];
      o[n][2] *= corr[1];
      o[n][3] *= corr[1];
    }
    // P * V over this warp's 128 value dims
#pragma unroll
    for (int kk = 0; kk < TILE / 16; ++kk) {
#pragma unroll
      for (int n2 = 0; n2 < NT / 2; ++n2) {
        const int j = lane >> 3, r = lane & 7;
        const int row = kk * 16 + (j & 1) * 8 + r;
        const int ch = warp * (VD / 8) + n2 * 2 + (j >> 1);
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(smem_u32(ts + swz(row, ch)), b0, b1, b2, b3);
        mma16816(o[2 * n2], pa[kk], b0, b1);
        mma16816(o[2 * n2 + 1], pa[kk], b2, b3);
      }
    }
    __syncthreads();  // tile and s_part are reused by the next iteration
  }
  cp_async_wait<0>();

  // every warp holds the same (m, l); it writes its own value dims
#pragma unroll
  for (int rr = 0; rr < 2; ++rr) {
    const int head = hg * 16 + g + rr * 8;
    if (head >= p.heads) continue;
    const float L = l_run[rr];
    const float inv = p.splits == 1 ? row_factor(p, t, head, m_run[rr], L) : L > 0.f ? 1.f / L : 0.f;
    const int d0 = warp * VD + 2 * t4;
    if (p.splits == 1) {
      bf16* dst = p.out + t * p.o_tok + head * p.o_head + d0;
#pragma unroll
      for (int n = 0; n < NT; ++n)
        if (d0 + n * 8 < pc) *reinterpret_cast<uint32_t*>(dst + n * 8) = pack_bf16(o[n][rr * 2] * inv, o[n][rr * 2 + 1] * inv);
    } else {
      const long long unit = (long long)t * p.heads + head;
      float* dst = p.part_o + (unit * p.splits + split) * pc + d0;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        if (d0 + n * 8 < pc) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[n][rr * 2] * inv, o[n][rr * 2 + 1] * inv);
      }
      if (warp == 0 && t4 == 0) p.part_lse[unit * p.splits + split] = L > 0.f ? m_run[rr] + log2f(L) : NEG_BIG;
    }
  }
}

template <int C>
__global__ void __launch_bounds__(128) mla_merge_kernel(const MlaParams p) {
  PG_PDL_ENTRY();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long unit = (long long)blockIdx.x * 4 + warp;  // (token, head)
  if (unit >= (long long)p.tokens * p.heads) return;
  const int t = (int)(unit / p.heads), head = (int)(unit % p.heads);
  const float* lse = p.part_lse + unit * p.splits;
  float M = NEG_BIG;
  for (int s = 0; s < p.splits; ++s) M = fmaxf(M, lse[s]);
  float acc[C / 32];
#pragma unroll
  for (int i = 0; i < C / 32; ++i) acc[i] = 0.f;
  float Wsum = 0.f;
  for (int s = 0; s < p.splits; ++s) {
    if (lse[s] <= NEG_BIG) continue;
    const float f = exp2f(lse[s] - M);
    Wsum += f;
    const float* po = p.part_o + (unit * p.splits + s) * p.c;
#pragma unroll
    for (int i = 0; i < C / 32; ++i)
      if (lane + 32 * i < p.c) acc[i] += f * po[lane + 32 * i];
  }
  bf16* dst = p.out + t * p.o_tok + head * p.o_head;
  const float inv = row_factor(p, t, head, M, Wsum);
#pragma unroll
  for (int i = 0; i < C / 32; ++i)
    if (lane + 32 * i < p.c) dst[lane + 32 * i] = __float2bfloat16(acc[i] * inv);
}

// One CTA per token.  z row: [.. zq: qr ..][.. zkv: c + r ..] inside one fused projection row.
template <typename T, int V>
__global__ void __launch_bounds__(256) latent_rows_kernel(const T* __restrict__ zq, const T* __restrict__ zkv, long long ld, const float* __restrict__ q_w, const float* __restrict__ kv_w,
                                                          const float* __restrict__ cos, const float* __restrict__ sin, const int* __restrict__ positions, const int* __restrict__ slots,
                                                          T* __restrict__ cq, T* __restrict__ latent, int qr, int c, int r, int max_pos, long long num_slots, float eps, uint32_t* status) {
  PG_PDL_ENTRY();
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const int tid = threadIdx.x;
  const T* qrow = zq + t * ld;
  const T* krow = zkv + t * ld;
  auto square_sum = [&](const T* row, int n) {
    float ss = 0.f;
    for (int i = tid; i < n / V; i += 256) {
      float f[V];
      load_vec<V>(row + i * V, f);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += f[j] * f[j];
    }
    return block_sum(ss, red);
  };
  auto write_norm = [&](const T* row, const float* w, T* dst, int n, float inv) {
    for (int i = tid; i < n / V; i += 256) {
      float f[V], wf[V];
      load_vec<V>(row + i * V, f);
      load_vec<V>(w + i * V, wf);
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] = f[j] * inv * wf[j];
      store_vec<V>(dst + i * V, f);
    }
  };
  if (qr > 0) {
    const float iq = rsqrtf(square_sum(qrow, qr) / (float)qr + eps);
    write_norm(qrow, q_w, cq + t * qr, qr, iq);
  }
  const float ik = rsqrtf(square_sum(krow, c) / (float)c + eps);
  const long long slot = slots[t];
  if (slot < 0 || slot >= num_slots) {
    if (tid == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (54u << 8));
    return;
  }
  T* dst = latent + slot * (c + r);
  write_norm(krow, kv_w, dst, c, ik);
  if (r > 0) {
    int pos = positions[t];
    if (pos < 0 || pos >= max_pos) {
      if (tid == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (55u << 8));
      pos = pos < 0 ? 0 : max_pos - 1;
    }
    for (int i = tid; i < r / 2; i += 256) {
      const float u = to_f32(krow[c + 2 * i]), v = to_f32(krow[c + 2 * i + 1]);
      const float cs = cos[(long long)pos * (r / 2) + i], sn = sin[(long long)pos * (r / 2) + i];
      dst[c + 2 * i] = from_f32<T>(u * cs - v * sn);
      dst[c + 2 * i + 1] = from_f32<T>(v * cs + u * sn);
    }
  }
}

// x[t, h, 0 .. r) in place, by strides; one thread per pair
template <typename T>
__global__ void __launch_bounds__(256) rotate_pairs_kernel(T* __restrict__ x, long long tok, long long head, const float* __restrict__ cos, const float* __restrict__ sin, const int* __restrict__ positions,
                                                           int tokens, int heads, int r, int max_pos) {
  PG_PDL_ENTRY();
  const int half = r / 2;
  const long long n = (long long)tokens * heads * half;
  for (long long e = (long long)blockIdx.x * 256 + threadIdx.x; e < n; e += (long long)gridDim.x * 256) {
    const int i = (int)(e % half), h = (int)(e / half % heads);
    const long long t = e / half / heads;
    const int pos = min(max(positions[t], 0), max_pos - 1);
    T* p = x + t * tok + h * head + 2 * i;
    const float u = to_f32(p[0]), v = to_f32(p[1]), cs = cos[(long long)pos * half + i], sn = sin[(long long)pos * half + i];
    p[0] = from_f32<T>(u * cs - v * sn);
    p[1] = from_f32<T>(v * cs + u * sn);
  }
}

constexpr int PL_KEYS = 128;  // keys per chunk, one per thread
constexpr int PL_VMAX = 16;   // latent columns per thread: c <= 2048

// One CTA per (query row, head); strides as in MlaParams, the queries' rotary part is turned here.
template <typename T>
__global__ void __launch_bounds__(128) latent_attention_plain_kernel(const T* __restrict__ q_abs, long long q_tok, long long q_head, const T* __restrict__ q_pe, long long pe_tok, long long pe_head,
                                                                     const float* __restrict__ cos, const float* __restrict__ sin, int max_pos, const T* __restrict__ latent, T* __restrict__ out,
                                                                     long long o_tok, long long o_head, const int* __restrict__ q_indptr, const int* __restrict__ kv_lens, const int* __restrict__ table,
                                                                     int table_stride, const int* __restrict__ unit_seq, int c, int r, int page_size, float scale, int window, const float* __restrict__ sink,
                                                                     const T* __restrict__ gate, long long ld_gate) {
  PG_PDL_ENTRY();
  extern __shared__ __align__(16) float sm[];
  const int w = c + r;
  float* sq = sm;        // [c + r]
  float* sp = sm + w;    // [PL_KEYS]
  __shared__ float red[4];
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int b = unit_seq[t];
  const int kv_len = kv_lens[b];
  const int n = kv_len == 0 ? 0 : kv_len - (q_indptr[b + 1] - 1 - t);  // keys up to the row's own
  const int first = window > 0 ? max(0, n - window) : 0;
  const int* pages = table + (long long)b * table_stride;
  for (int i = tid; i < c; i += 128) sq[i] = to_f32(q_abs[t * q_tok + h * q_head + i]);
  for (int i = tid; i < r / 2; i += 128) {
    const T* p = q_pe + t * pe_tok + h * pe_head + 2 * i;
    const long long at = (long long)min(max(n - 1, 0), max_pos - 1) * (r / 2) + i;
    const float u = to_f32(p[0]), v = to_f32(p[1]), cs = cos[at], sn = sin[at];
    sq[c + 2 * i] = u * cs - v * sn;
    sq[c + 2 * i + 1] = v * cs + u * sn;
  }
  __syncthreads();
  float m = -INFINITY, l = 0.f, acc[PL_VMAX];
#pragma unroll
  for (int i = 0; i < PL_VMAX; ++i) acc[i] = 0.f;
  for (int k0 = first; k0 < n; k0 += PL_KEYS) {
    const int key = k0 + tid;
    float s = -INFINITY;
    if (key < n) {
      const T* kr = latent + ((long long)pages[key / page_size] * page_size + key % page_size) * w;
      float a = 0.f;
      for (int i = 0; i < w; ++i) a = fmaf(sq[i], to_f32(kr[i]), a);
      s = a * scale;
    }
    float mx = warp_max(s);
    if (lane == 0) red[warp] = mx;
    __syncthreads();
    mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    const float m_new = fmaxf(m, mx);
    const float p = key < n ? __expf(s - m_new) : 0.f;
    sp[tid] = p;
    const float ps = warp_sum(p);
    __syncthreads();  // everyone has read the maxima
    if (lane == 0) red[warp] = ps;
    __syncthreads();
    const float corr = m == -INFINITY ? 0.f : __expf(m - m_new);
    l = l * corr + ((red[0] + red[1]) + (red[2] + red[3]));
    m = m_new;
    const int cnt = min(PL_KEYS, n - k0);
#pragma unroll
    for (int i = 0; i < PL_VMAX; ++i) acc[i] *= corr;
    for (int j = 0; j < cnt; ++j) {
      const int kk = k0 + j;
      const T* vr = latent + ((long long)pages[kk / page_size] * page_size + kk % page_size) * w;
      const float pj = sp[j];
#pragma unroll
      for (int i = 0; i < PL_VMAX; ++i)
        if (tid + 128 * i < c) acc[i] = fmaf(pj, to_f32(vr[tid + 128 * i]), acc[i]);
    }
    __syncthreads();
  }
  if (sink && l > 0.f) l += __expf(sink[h] - m);
  float f = l > 0.f ? 1.f / l : 0.f;
  if (gate) f /= 1.f + __expf(-to_f32(gate[t * ld_gate + h]));
#pragma unroll
  for (int i = 0; i < PL_VMAX; ++i)
    if (tid + 128 * i < c) out[t * o_tok + h * o_head + tid + 128 * i] = from_f32<T>(acc[i] * f);
}

template <int C, int R, bool EXACT>
int launch_mla(const MlaParams& p, cudaStream_t stream) {
  constexpr size_t smem = (size_t)2 * 32 * (C + R) * 2 + 4 * 16 * 32 * 4;
  static bool set = false;
  if (!set) {
    PG_CUDA(cudaFuncSetAttribute(mla_attn_kernel<C, R, EXACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    set = true;
  }
  const int grid = p.tokens * ((p.heads + 15) / 16) * p.splits;
  PG_CUDA(launch_pdl(mla_attn_kernel<C, R, EXACT>, dim3((unsigned)grid), dim3(128), smem, stream, p));
  PG_LAUNCH_CHECK();
  if (p.splits > 1) {
    PG_CUDA(launch_pdl(mla_merge_kernel<C>, dim3((unsigned)(((long long)p.tokens * p.heads + 3) / 4)), dim3(128), (size_t)0, stream, p));
    PG_LAUNCH_CHECK();
  }
  return PG_OK;
}

}  // namespace

extern "C" int pg_mla_append(const void* kv_a, long long ld, const void* norm_w, const void* cos, const void* sin, const void* positions,
                             const void* slots, void* latent, int tokens, int c, int rope, int max_pos, long long num_slots, float eps,
                             void* status, cudaStream_t stream) {
  if (tokens == 0) return PG_OK;
  mla_append_kernel<<<(tokens + 3) / 4, 128, 0, stream>>>((const bf16*)kv_a, ld, (const bf16*)norm_w, (const bf16*)cos, (const bf16*)sin,
                                                         (const int*)positions, (const int*)slots, (bf16*)latent, tokens, c, rope, max_pos,
                                                         num_slots, eps, (uint32_t*)status);
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_mla_q_prep(const void* q, const void* cos, const void* sin, const void* positions, void* q_nope_hm, void* q_pe, int tokens,
                             int heads, int nope, int rope, int max_pos, cudaStream_t stream) {
  PG_REQUIRE(nope % 8 == 0 && rope % 2 == 0, "mla_q_prep: nope %d / rope %d not supported", nope, rope);
  if (tokens == 0) return PG_OK;
  const long long units = (long long)tokens * heads;
  mla_q_prep_kernel<<<(unsigned)((units + 3) / 4), 128, 0, stream>>>((const bf16*)q, (const bf16*)cos, (const bf16*)sin, (const int*)positions,
                                                                    (bf16*)q_nope_hm, (bf16*)q_pe, tokens, heads, nope, rope, max_pos);
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_permute_021(const void* in, void* out, int A, int B, int D, cudaStream_t stream) {
  PG_REQUIRE(D % 8 == 0, "permute: inner dim %d must be a multiple of 8", D);
  if ((long long)A * B == 0) return PG_OK;
  permute_021_kernel<<<(unsigned)((long long)A * B), 64, 0, stream>>>((const bf16*)in, (bf16*)out, A, B, D);
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_mla_attention(const void* q_abs, const void* q_pe, const void* latent, void* out, const void* q_indptr, const void* kv_lens,
                                const void* table, int table_stride, const void* unit_seq, int num_seqs, int tokens, int heads, int c, int rope,
                                int page_size, float scale, int splits, void* part_o, void* part_lse, void* status, cudaStream_t stream) {
  PG_REQUIRE(c == 512 && rope == 64, "mla_attention: built for kv_lora 512 + rope 64 (got %d + %d)", c, rope);
  PG_REQUIRE(heads % 16 == 0, "mla_attention: heads %d must be a multiple of 16", heads);
  // head-major absorbed queries and outputs, token-major rotated query parts
  return pg_latent_attention(q_abs, c, (long long)tokens * c, q_pe, (long long)heads * rope, rope, nullptr, nullptr, 0, latent, out, c, (long long)tokens * c, q_indptr, kv_lens, table, table_stride, unit_seq, 0,
                             num_seqs, tokens, heads, c, rope, page_size, scale, 0, nullptr, nullptr, 0, splits, part_o, part_lse, stream);
}

// q_abs, q_pe and out by token / head strides in elements; cos / sin f32 [max_pos, r / 2] turn the q_pe columns (null: they
// come rotated); window > 0: a row sees its last `window` keys; sink f32 [heads] and head_gate bf16 [tokens, >= heads] as in
// MlaParams (or null).  Row 0 of this call is row `first_row` of the step that q_indptr and unit_seq describe.
extern "C" int pg_latent_attention(const void* q_abs, long long q_tok, long long q_head, const void* q_pe, long long pe_tok, long long pe_head, const void* cos, const void* sin, int max_pos,
                                   const void* latent, void* out, long long o_tok, long long o_head, const void* q_indptr, const void* kv_lens, const void* table, int table_stride,
                                   const void* unit_seq, int first_row, int num_seqs, int tokens, int heads, int c, int r, int page_size, float scale, int window, const void* sink, const void* head_gate, long long ld_gate,
                                   int splits, void* part_o, void* part_lse, cudaStream_t stream) {
  PG_REQUIRE(c % 8 == 0 && r % 8 == 0 && c >= 8 && c <= 512 && r >= 0 && r <= 64, "latent_attention: a latent of %d + %d columns is not supported (multiples of 8 up to 512 + 64)", c, r);
  PG_REQUIRE(page_size == 16 || page_size == 32 || page_size == 64, "latent_attention: pages of %d tokens", page_size);
  PG_REQUIRE(q_tok % 2 == 0 && q_head % 2 == 0 && pe_tok % 2 == 0 && pe_head % 2 == 0 && o_tok % 2 == 0 && o_head % 2 == 0, "latent_attention: strides must keep column pairs aligned");
  PG_REQUIRE((cos == nullptr) == (sin == nullptr) && (cos == nullptr || max_pos > 0), "latent_attention: rotation tables come together");
  if (tokens == 0) return PG_OK;
  MlaParams p;
  p.q_abs = (const bf16*)q_abs, p.q_tok = q_tok, p.q_head = q_head;
  p.q_pe = (const bf16*)q_pe, p.pe_tok = pe_tok, p.pe_head = pe_head;
  p.cos = (const float*)cos, p.sin = (const float*)sin, p.max_pos = max_pos;
  p.latent = (const bf16*)latent;
  p.out = (bf16*)out, p.o_tok = o_tok, p.o_head = o_head;
  p.c = c, p.r = r, p.window = window;
  p.sink = (const float*)sink, p.gate = (const bf16*)head_gate, p.ld_gate = ld_gate;
  p.q_indptr = (const int*)q_indptr;
  p.kv_lens = (const int*)kv_lens;
  p.table = (const int*)table;
  p.table_stride = table_stride;
  p.num_seqs = num_seqs;
  p.tokens = tokens;
  p.heads = heads;
  p.page_size = page_size;
  p.splits = splits < 1 ? 1 : splits;
  p.scale_log2 = scale * LOG2E;
  p.part_o = (float*)part_o;
  p.part_lse = (float*)part_lse;
  p.unit_seq = (const int*)unit_seq;
  p.first_row = first_row;
  PG_REQUIRE(p.splits == 1 || (part_o && part_lse), "latent_attention: split-KV needs partial buffers");
  if (c == 512 && r == 64) return launch_mla<512, 64, true>(p, stream);
  if (c == 512 && r == 0) return launch_mla<512, 0, true>(p, stream);
  if (c <= 128) return r ? launch_mla<128, 64, false>(p, stream) : launch_mla<128, 0, false>(p, stream);
  if (c <= 256) return r ? launch_mla<256, 64, false>(p, stream) : launch_mla<256, 0, false>(p, stream);
  return r ? launch_mla<512, 64, false>(p, stream) : launch_mla<512, 0, false>(p, stream);
}

extern "C" int pg_latent_attention_plain(const void* q_abs, long long q_tok, long long q_head, const void* q_pe, long long pe_tok, long long pe_head, const void* cos, const void* sin, int max_pos,
                                         const void* latent, void* out, long long o_tok, long long o_head, const void* q_indptr, const void* kv_lens, const void* table, int table_stride,
                                         const void* unit_seq, int tokens, int heads, int c, int r, int page_size, float scale, int window, const void* sink, const void* head_gate, long long ld_gate, int is_f32,
                                         cudaStream_t stream) {
  PG_REQUIRE(c >= 1 && c <= 128 * PL_VMAX && r >= 0 && r % 2 == 0 && r <= 2048 && heads <= 65535, "latent_attention_plain: %d heads over %d + %d columns", heads, c, r);
  PG_REQUIRE(r == 0 || (cos && sin && max_pos > 0), "latent_attention_plain: rotated columns need their tables");
  if (tokens == 0) return PG_OK;
  const size_t smem = (size_t)(c + r + PL_KEYS) * 4;
#define PG_LAP(T)                                                                                                                                                                                   \
  launch_pdl(latent_attention_plain_kernel<T>, dim3(tokens, heads), dim3(128), smem, stream, (const T*)q_abs, q_tok, q_head, (const T*)q_pe, pe_tok, pe_head, (const float*)cos, (const float*)sin, \
             max_pos, (const T*)latent, (T*)out, o_tok, o_head, (const int*)q_indptr, (const int*)kv_lens, (const int*)table, table_stride, (const int*)unit_seq, c, r, page_size, scale, window, \
             (const float*)sink, (const T*)head_gate, ld_gate)
  PG_CUDA(is_f32 ? PG_LAP(float) : PG_LAP(bf16));
#undef PG_LAP
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_latent_rows(const void* zq, const void* zkv, long long ld, const void* q_w, const void* kv_w, const void* cos, const void* sin, const void* positions, const void* slots, void* cq,
                              void* latent, int tokens, int qr, int c, int r, int max_pos, long long num_slots, float eps, int is_f32, void* status, cudaStream_t stream) {
  PG_REQUIRE(qr >= 0 && c >= 1 && r >= 0 && r % 2 == 0 && (r == 0 || (cos && sin && max_pos > 0)), "latent_rows: sizes %d, %d + %d", qr, c, r);
  if (tokens == 0) return PG_OK;
  const bool v8 = !is_f32 && qr % 8 == 0 && c % 8 == 0 && r % 8 == 0 && ld % 8 == 0 && (((uintptr_t)zq | (uintptr_t)zkv | (uintptr_t)q_w | (uintptr_t)kv_w | (uintptr_t)cq | (uintptr_t)latent) & 15) == 0;
#define PG_LR(T, V)                                                                                                                                                                                \
  launch_pdl(latent_rows_kernel<T, V>, dim3(tokens), dim3(256), (size_t)0, stream, (const T*)zq, (const T*)zkv, ld, (const float*)q_w, (const float*)kv_w, (const float*)cos, (const float*)sin,   \
             (const int*)positions, (const int*)slots, (T*)cq, (T*)latent, qr, c, r, max_pos, num_slots, eps, (uint32_t*)status)
  if (is_f32)
    PG_CUDA(PG_LR(float, 1));
  else
    PG_CUDA(v8 ? PG_LR(bf16, 8) : PG_LR(bf16, 1));
#undef PG_LR
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_rotate_pairs(void* x, long long tok, long long head, const void* cos, const void* sin, const void* positions, int tokens, int heads, int r, int max_pos, int is_f32, cudaStream_t stream) {
  PG_REQUIRE(r % 2 == 0 && max_pos > 0, "rotate_pairs: %d columns", r);
  long long blocks = ((long long)tokens * heads * (r / 2) + 255) / 256;
  if (blocks == 0) return PG_OK;
  if (blocks > 148 * 32) blocks = 148 * 32;
#define PG_RP(T) launch_pdl(rotate_pairs_kernel<T>, dim3((unsigned)blocks), dim3(256), (size_t)0, stream, (T*)x, tok, head, (const float*)cos, (const float*)sin, (const int*)positions, tokens, heads, r, max_pos)
  PG_CUDA(is_f32 ? PG_RP(float) : PG_RP(bf16));
#undef PG_RP
  PG_LAUNCH_CHECK();
  return PG_OK;
}
