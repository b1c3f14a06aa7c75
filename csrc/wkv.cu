// Linear attention with a decay per token and key channel (WKV): the token shift in front of its projections, and the
// recurrence in blocks of 16 tokens on the tensor cores.
//
//  * token_mix: every projection of the layer reads its own mix of a token's row with the previous one's,
//      out[t, i] = h[t] + (h[t - 1] - h[t]) * mu[i].
//    The row in front of a step's first row comes from the request's slot, which then takes the step's last row.  A thread
//    owns V columns for a run of rows, so the mix weights stay in registers and each row is read once.
//  * wkv_block: o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t, S_t = diag(w_t) S_(t-1) + k_t v_t^T over blocks of 16 tokens.  With S0
//    the state in front of a block and products of decays over tokens of the block,
//      O = (R diag(prod_(i < t) w_i)) S0 + A V,   A_ts = sum_d r_t k_s prod_(s < i < t) w_i  (s < t),   A_tt = sum_d r_t u k_t,
//      S1 = diag(prod_i w_i) S0 + (K diag(prod_(i > s) w_i))^T V.
//    Every factor is a product of numbers in (0, 1), so nothing overflows however strong the decay is.
//    A CTA takes 64 value columns of one (sequence, head).  Four warps keep the transposed state, 16 value columns each, in
//    f32 accumulators for the whole sequence: as the A operand of the next block's product they are used where they are.
//    The other warps make the next block's operands meanwhile, one thread per key channel and half of the pairs (t, s): raw
//    rows arrive by cp.async two blocks ahead, the products run along the block, the sums over channels of the 136 entries of
//    A are folded by shuffles, 32 at a time.  What is formed in 32 bits and multiplied again (the state, the decayed R and K,
//    A) enters the tensor cores as the sum of two bf16 numbers.
#include "api.h"
#include "common.cuh"
#include "mma_frag.cuh"
#include "types.cuh"

namespace {

// N: the number of mixes rounded up to an instantiated size; a CTA takes `run` rows.
template <typename T, int V, int N>
__global__ void __launch_bounds__(128) token_mix_kernel(const T* __restrict__ h, long long ldh, const float* __restrict__ mu, T* __restrict__ carried, T* __restrict__ out, const int* __restrict__ unit_seq,
                                                        const int* __restrict__ q_indptr, const int* __restrict__ slots, int tokens, int n, int width, int run) {
  PG_PDL_ENTRY();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= width) return;
  const int t0 = blockIdx.y * run, t1 = min(tokens, t0 + run);
  float m[N][V];
#pragma unroll
  for (int i = 0; i < N; ++i)
    if (i < n) load_vec<V>(mu + (long long)i * width + c, m[i]);
  float back[V], own[V];
  if (t0 > 0) load_vec<V>(h + (t0 - 1) * ldh + c, back);  // in front of a sequence's first row it is replaced below
  for (int t = t0; t < t1; ++t) {
    const int b = unit_seq[t];
    load_vec<V>(h + t * ldh + c, own);
    if (t == q_indptr[b]) {
      const int slot = slots[b];
      if (slot >= 0) {
        T* st = carried + (long long)slot * width + c;
        load_vec<V>(st, back);
        float last[V];
        load_vec<V>(h + (long long)(q_indptr[b + 1] - 1) * ldh + c, last);
        store_vec<V>(st, last);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) back[j] = 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (i < n) {
        float o[V];
#pragma unroll
        for (int j = 0; j < V; ++j) o[j] = fmaf(back[j] - own[j], m[i][j], own[j]);
        store_vec<V>(out + ((long long)t * n + i) * width + c, o);
      }
#pragma unroll
    for (int j = 0; j < V; ++j) back[j] = own[j];
  }
}

// ---- wkv_block -------------------------------------------------------------------------
constexpr int BT = 16;         // tokens per block
constexpr int DVC = 64;        // value columns per CTA
constexpr int LDA = BT + 8;    // row pitch of the 16-column tiles
constexpr int PAIRS0 = 72, PAIRS1 = 64;  // entries of A that the two halves of the operand threads sum

__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const float ah = bf16_round(a), bh = bf16_round(b);
  hi = pack2(ah, bh);
  lo = pack2(a - ah, b - bh);
}

template <int DK>
struct WkvSmem {
  static constexpr int LDK = DK + 8;
  float f[2][BT * DK];                                            // raw decay projection of the coming blocks
  bf16 r[2][BT * DK], k[2][BT * DK];
  bf16 rt_hi[2][BT * LDK], rt_lo[2][BT * LDK], kt_hi[2][BT * LDK], kt_lo[2][BT * LDK];
  bf16 a_hi[2][BT * LDA], a_lo[2][BT * LDA];
  bf16 v[4][2][BT * LDA], o[4][BT * LDA];                         // private to a state warp
  float dec[2][DK];
  float part0[DK / 32][PAIRS0], part1[DK / 32][PAIRS1];           // sums over 32 channels
};

// val[i] summed over the warp's lanes: lane l gets the sum of val[l].
__device__ __forceinline__ float fold32(float (&val)[32], int lane) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? val[i] : val[i + o], keep = up ? val[i + o] : val[i];
      val[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  return val[0];
}

// Sums over a warp's 32 channels of the entries of A with s even (HALF 0; and the diagonal's first half) or odd (HALF 1; and the
// diagonal's second half), in the order that pair_of undoes.
template <int HALF>
__device__ __forceinline__ void sum_pairs(const float (&r)[BT], const float (&k)[BT], const float (&w)[BT], float u, int lane, float* part) {
  float val[32];
  int n = 0;
#pragma unroll
  for (int s = HALF; s < BT - 1; s += 2) {
    float q = k[s];
#pragma unroll
    for (int t = s + 1; t < BT; ++t) {
      val[n & 31] = r[t] * q;
      q *= w[t];
      if ((++n & 31) == 0) part[n - 32 + lane] = fold32(val, lane);
    }
  }
#pragma unroll
  for (int t = 0; t < 8; ++t) val[(n + t) & 31] = r[HALF * 8 + t] * u * k[HALF * 8 + t];
  if (HALF) {
    part[32 + lane] = fold32(val, lane);
  } else {
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {
      const bool up = lane & o;
#pragma unroll
      for (int i = 0; i < o; ++i) {
        const float send = up ? val[i] : val[i + o], keep = up ? val[i + o] : val[i];
        val[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
    }
    val[0] += __shfl_xor_sync(0xffffffffu, val[0], 8);
    val[0] += __shfl_xor_sync(0xffffffffu, val[0], 16);
    if (lane < 8) part[64 + lane] = val[0];
  }
}

// Place in A (t * LDA + s) of entry `j` of the two lists, one behind the other.
__device__ __forceinline__ int pair_of(int j) {
  const int half = j >= PAIRS0;
  int n = half ? j - PAIRS0 : j;
  for (int s = half; s < BT - 1; s += 2) {
    if (n < BT - 1 - s) return (s + 1 + n) * LDA + s;
    n -= BT - 1 - s;
  }
  return (half * 8 + n) * (LDA + 1);
}

template <int DK>
__global__ void __launch_bounds__(128 + 2 * DK) wkv_block_kernel(const bf16* __restrict__ r, const bf16* __restrict__ k, const bf16* __restrict__ v, long long ld, const float* __restrict__ f, long long ldf,
                                                                 const float* __restrict__ w0, const float* __restrict__ u, float* __restrict__ state, bf16* __restrict__ out, const int* __restrict__ q_indptr,
                                                                 const int* __restrict__ slots, int heads, int dk, int dv, int col_blocks, int min_len) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  WkvSmem<DK>& sm = *reinterpret_cast<WkvSmem<DK>*>(smem_raw);
  constexpr int LDK = WkvSmem<DK>::LDK;
  const int h = blockIdx.x / col_blocks, dv0 = (blockIdx.x % col_blocks) * DVC, b = blockIdx.y;
  const int slot = slots[b], q0 = q_indptr[b], q1 = q_indptr[b + 1];
  if (q1 == q0 || q1 - q0 < min_len || slot < 0) return;
  const int blocks = (q1 - q0 + BT - 1) / BT;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int i = tid; i < 2 * BT * LDA; i += 128 + 2 * DK) (&sm.a_hi[0][0])[i] = (&sm.a_lo[0][0])[i] = __float2bfloat16(0.f);  // above the diagonal
  __syncthreads();

  if (warp < 4) {
    // ---- state: rows = value columns m0 + g, m0 + g + 8, columns = key channels -----------------------------
    const int g = lane >> 2, t4 = lane & 3, m0 = dv0 + warp * 16;
    float* S = state + ((long long)slot * heads + h) * dk * dv;
    float s[DK / 8][4];
#pragma unroll
    for (int j = 0; j < DK / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = j * 8 + 2 * t4 + (e & 1), c = m0 + g + (e >> 1) * 8;
        s[j][e] = d < dk && c < dv ? S[(long long)d * dv + c] : 0.f;
      }
    const int vr = lane >> 1, vc = (lane & 1) * 8;  // the lane's 16 bytes of a value or output tile
    const bool in = m0 + vc < dv;
    auto load_v = [&](int blk) {
      const int t = q0 + blk * BT + vr;
      const bool ok = in && t < q1;
      cp_async16(&sm.v[warp][blk & 1][vr * LDA + vc], v + (long long)(ok ? t : q0) * ld + (long long)h * dv + (ok ? m0 + vc : 0), ok);
      cp_async_commit();
    };
    load_v(0);
    __syncthreads();
    for (int blk = 0; blk < blocks; ++blk) {
      const int buf = blk & 1;
      cp_async_wait_all();
      __syncwarp();
      uint32_t va[4], x[4];
      frag_a_t(sm.v[warp][buf], LDA, 0, 0, lane, va);
      if (blk + 1 < blocks) load_v(blk + 1);
      float o[2][4] = {};
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        uint32_t hi[4], lo[4];
        split2(s[2 * ks][0], s[2 * ks][1], hi[0], lo[0]);
        split2(s[2 * ks][2], s[2 * ks][3], hi[1], lo[1]);
        split2(s[2 * ks + 1][0], s[2 * ks + 1][1], hi[2], lo[2]);
        split2(s[2 * ks + 1][2], s[2 * ks + 1][3], hi[3], lo[3]);
        frag_b_nk(sm.rt_hi[buf], LDK, 0, ks * 16, lane, x);
        mma16816(o[0], hi, x[0], x[1]);
        mma16816(o[1], hi, x[2], x[3]);
        mma16816(o[0], lo, x[0], x[1]);
        mma16816(o[1], lo, x[2], x[3]);
        frag_b_nk(sm.rt_lo[buf], LDK, 0, ks * 16, lane, x);
        mma16816(o[0], hi, x[0], x[1]);
        mma16816(o[1], hi, x[2], x[3]);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const float2 d = *reinterpret_cast<const float2*>(&sm.dec[buf][(2 * ks + n) * 8 + 2 * t4]);
          s[2 * ks + n][0] *= d.x, s[2 * ks + n][1] *= d.y, s[2 * ks + n][2] *= d.x, s[2 * ks + n][3] *= d.y;
        }
        frag_b_kn(sm.kt_hi[buf], LDK, 0, ks * 16, lane, x);
        mma16816(s[2 * ks], va, x[0], x[1]);
        mma16816(s[2 * ks + 1], va, x[2], x[3]);
        frag_b_kn(sm.kt_lo[buf], LDK, 0, ks * 16, lane, x);
        mma16816(s[2 * ks], va, x[0], x[1]);
        mma16816(s[2 * ks + 1], va, x[2], x[3]);
      }
      frag_b_nk(sm.a_hi[buf], LDA, 0, 0, lane, x);
      mma16816(o[0], va, x[0], x[1]);
      mma16816(o[1], va, x[2], x[3]);
      frag_b_nk(sm.a_lo[buf], LDA, 0, 0, lane, x);
      mma16816(o[0], va, x[0], x[1]);
      mma16816(o[1], va, x[2], x[3]);
      bf16* ot = sm.o[warp];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) ot[(n * 8 + 2 * t4 + (e & 1)) * LDA + g + (e >> 1) * 8] = __float2bfloat16(o[n][e]);
      __syncwarp();
      const int t = q0 + blk * BT + vr;
      if (in && t < q1) *reinterpret_cast<uint4*>(out + ((long long)t * heads + h) * dv + m0 + vc) = *reinterpret_cast<const uint4*>(&ot[vr * LDA + vc]);
      __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < DK / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = j * 8 + 2 * t4 + (e & 1), c = m0 + g + (e >> 1) * 8;
        if (d < dk && c < dv) S[(long long)d * dv + c] = s[j][e];
      }
    return;
  }

  // ---- operands of the coming block -----------------------------------------------------------------------
  const int p = tid - 128, d = p % DK, half = p / DK, pw = d >> 5;
  const float w0d = d < dk ? w0[h * dk + d] : 0.f, ud = d < dk ? u[h * dk + d] : 0.f;
  const int place = p < PAIRS0 + PAIRS1 ? pair_of(p) : 0;
  auto bar = [] { asm volatile("bar.sync 1, %0;" ::"n"(2 * DK) : "memory"); };
  auto load_raw = [&](int blk) {
    const int t0 = q0 + blk * BT, st = blk & 1;
#pragma unroll
    for (int c = p; c < BT * (DK / 4); c += 2 * DK) {
      const int t = c / (DK / 4), e = c % (DK / 4) * 4;
      const bool ok = t0 + t < q1 && e < dk;
      cp_async16(&sm.f[st][t * DK + e], f + (long long)(ok ? t0 + t : q0) * ldf + (long long)h * dk + (ok ? e : 0), ok);
    }
#pragma unroll
    for (int c = p; c < BT * (DK / 8); c += 2 * DK) {
      const int t = c / (DK / 8), e = c % (DK / 8) * 8;
      const bool ok = t0 + t < q1 && e < dk;
      const long long at = (long long)(ok ? t0 + t : q0) * ld + (long long)h * dk + (ok ? e : 0);
      cp_async16(&sm.r[st][t * DK + e], r + at, ok);
      cp_async16(&sm.k[st][t * DK + e], k + at, ok);
    }
    cp_async_commit();
  };
  auto make = [&](int blk) {
    const int buf = blk & 1, left = q1 - q0 - blk * BT;
    cp_async_wait_all();
    bar();  // the raw rows of this block are here
    if (blk + 1 < blocks) load_raw(blk + 1);
    float w[BT], rr[BT], kk[BT];
#pragma unroll
    for (int t = 0; t < BT; ++t) {
      w[t] = t < left ? __expf(-__expf(sm.f[buf][t * DK + d] + w0d)) : 1.f;  // rows past the end leave the state as it is
      rr[t] = __bfloat162float(sm.r[buf][t * DK + d]);
      kk[t] = __bfloat162float(sm.k[buf][t * DK + d]);
    }
    float x = 1.f;
    if (half == 0) {
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        const float y = rr[t] * x;
        const bf16 hi = __float2bfloat16(y);
        sm.rt_hi[buf][t * LDK + d] = hi;
        sm.rt_lo[buf][t * LDK + d] = __float2bfloat16(y - __bfloat162float(hi));
        x *= w[t];
      }
      sm.dec[buf][d] = x;
      sum_pairs<0>(rr, kk, w, ud, lane, sm.part0[pw]);
    } else {
#pragma unroll
      for (int t = BT - 1; t >= 0; --t) {
        const float y = kk[t] * x;
        const bf16 hi = __float2bfloat16(y);
        sm.kt_hi[buf][t * LDK + d] = hi;
        sm.kt_lo[buf][t * LDK + d] = __float2bfloat16(y - __bfloat162float(hi));
        x *= w[t];
      }
      sum_pairs<1>(rr, kk, w, ud, lane, sm.part1[pw]);
    }
    bar();
    for (int j = p; j < PAIRS0 + PAIRS1; j += 2 * DK) {
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < DK / 32; ++i) a += j < PAIRS0 ? sm.part0[i][j] : sm.part1[i][j - PAIRS0];
      const int at = j == p ? place : pair_of(j);
      const bf16 hi = __float2bfloat16(a);
      sm.a_hi[buf][at] = hi;
      sm.a_lo[buf][at] = __float2bfloat16(a - __bfloat162float(hi));
    }
  };
  load_raw(0);
  make(0);
  __syncthreads();
  for (int blk = 0; blk < blocks; ++blk) {
    if (blk + 1 < blocks) make(blk + 1);
    __syncthreads();
  }
}

template <int DK>
int launch_wkv_block(const void* r, const void* k, const void* v, long long ld, const void* f, long long ldf, const void* w0, const void* u, void* state, void* out, const void* q_indptr, const void* slots,
                     int num_seqs, int heads, int dk, int dv, int min_len, cudaStream_t stream) {
  static bool set = false;
  if (!set) {
    PG_CUDA(cudaFuncSetAttribute(wkv_block_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(WkvSmem<DK>)));
    set = true;
  }
  const int cb = (dv + DVC - 1) / DVC;
  wkv_block_kernel<DK><<<dim3(heads * cb, num_seqs), 128 + 2 * DK, sizeof(WkvSmem<DK>), stream>>>((const bf16*)r, (const bf16*)k, (const bf16*)v, ld, (const float*)f, ldf, (const float*)w0, (const float*)u,
                                                                                                 (float*)state, (bf16*)out, (const int*)q_indptr, (const int*)slots, heads, dk, dv, cb, min_len);
  PG_LAUNCH_CHECK();
  return PG_OK;
}

}  // namespace

extern "C" int pg_wkv_block(const void* r, const void* k, const void* v, long long ld, const void* f, long long ldf, const void* w0, const void* u, void* state, void* out, const void* q_indptr,
                            const void* slots, int num_seqs, int heads, int dk, int dv, int min_len, cudaStream_t stream) {
  PG_REQUIRE(dk % 8 == 0 && dk >= 8 && dk <= 128 && dv % 8 == 0 && dv >= 8, "wkv_block: key width %d (a multiple of 8 up to 128), value width %d (a multiple of 8)", dk, dv);
  PG_REQUIRE(ld % 8 == 0 && ldf % 4 == 0 && (((uintptr_t)r | (uintptr_t)k | (uintptr_t)v | (uintptr_t)f | (uintptr_t)out) & 15) == 0, "wkv_block: rows must be 16-byte aligned");
  PG_REQUIRE(num_seqs <= 65535, "wkv_block: %d sequences", num_seqs);
  if (num_seqs == 0) return PG_OK;
  if (dk <= 64) return launch_wkv_block<64>(r, k, v, ld, f, ldf, w0, u, state, out, q_indptr, slots, num_seqs, heads, dk, dv, min_len, stream);
  return launch_wkv_block<128>(r, k, v, ld, f, ldf, w0, u, state, out, q_indptr, slots, num_seqs, heads, dk, dv, min_len, stream);
}

extern "C" int pg_token_mix(const void* h, long long ldh, const void* mu, void* carried, void* out, const void* unit_seq, const void* q_indptr, const void* slots, int tokens, int n, int width, int is_f32,
                            cudaStream_t stream) {
  PG_REQUIRE(n >= 1 && n <= 8 && width >= 1, "token_mix: %d mixes (1..8) of %d columns", n, width);
  if (tokens == 0) return PG_OK;
  const int es = is_f32 ? 4 : 2;
  auto ok = [&](int v) {
    return width % v == 0 && ldh % v == 0 && (((uintptr_t)h | (uintptr_t)carried | (uintptr_t)out) % (v * es)) == 0 && ((uintptr_t)mu % 16) == 0;
  };
  const int v = is_f32 ? (ok(4) ? 4 : 1) : ok(8) ? 8 : ok(4) ? 4 : 1;
  const int cols = (width + 128 * v - 1) / (128 * v);
  int run = 1;
  while (run < 16 && (long long)cols * ((tokens + 2 * run - 1) / (2 * run)) >= 148 * 8) run *= 2;  // longer runs once every SM has work
  const dim3 grid(cols, (tokens + run - 1) / run);
  PG_REQUIRE(grid.y <= 65535u, "token_mix: %d rows", tokens);
#define PG_TM(T, V, N)                                                                                                                                                                            \
  launch_pdl(token_mix_kernel<T, V, N>, grid, dim3(128), (size_t)0, stream, (const T*)h, ldh, (const float*)mu, (T*)carried, (T*)out, (const int*)unit_seq, (const int*)q_indptr, (const int*)slots, \
             tokens, n, width, run)
#define PG_TMN(T, V) (n <= 5 ? PG_TM(T, V, 5) : PG_TM(T, V, 8))
  if (is_f32)
    PG_CUDA(v == 4 ? PG_TMN(float, 4) : PG_TMN(float, 1));
  else
    PG_CUDA(v == 8 ? PG_TMN(bf16, 8) : v == 4 ? PG_TMN(bf16, 4) : PG_TMN(bf16, 1));
#undef PG_TMN
#undef PG_TM
  PG_LAUNCH_CHECK();
  return PG_OK;
}
