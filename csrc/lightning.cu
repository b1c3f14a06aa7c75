// Linear attention with one decay per head as a chunk-wise scan on the tensor cores: a fixed one (lightning attention), or one per
// token (state-space duality, SSD below).
//
//   S_t = d S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t      (q, k, v = SiLU of the projections, d the head's decay)
//
// over chunks of 64 tokens, with S0 the state in front of the chunk and n its number of tokens:
//   O  = diag(d^(i+1)) Q S0 + P V,   P_ij = d^(i-j) (q_i . k_j) for j <= i,
//   S1 = d^n S0 + K^T (diag(d^(n-1-j)) V).
// q, k and v are bf16 operands as they are (the activation's result is rounded to the activation type); everything that is
// formed from them in 32 bits and then multiplied again (the state, P, the decayed V) enters the tensor cores as the sum of
// two bf16 numbers, so a product keeps 16 bits of it, and all sums are f32.  The state itself stays in f32 registers, as the
// accumulator of the last product, for the whole sequence.
//
// SSD: with d = softplus(dt + dt_bias) per token and head and c_i the running sum of -exp(A_log) d in the chunk, d^(i-j) becomes
// exp(c_i - c_j), never a quotient of two small numbers, d_j multiplies row j of V (through P and the decayed V), D joins the
// diagonal of P, and q = C and k = B are rows of a group of heads, as they are.
//
// CTA = (sequence, head, 64 value columns); 8 warps; the raw rows of the next chunk arrive by cp.async in the other of two
// buffers and are turned into SiLU in place.  Sequences below min_len tokens (decode rows) run in pg_decay_recurrent.
#include "api.h"
#include "common.cuh"
#include "mma_frag.cuh"

namespace {

constexpr int C = 64;        // tokens per chunk
constexpr int DVC = 64;      // value columns per CTA
constexpr int LDV = DVC + 8;

template <int DK>
struct LightSmem {
  static constexpr int LDK = DK + 8;
  bf16 q[2][C * LDK], k[2][C * LDK], v[2][C * LDV];
  bf16 vd_hi[C * LDV], vd_lo[C * LDV];   // diag(d^(n-1-j)) V
  bf16 s_hi[DK * LDV], s_lo[DK * LDV];   // S0
  float pw[C + 1];                       // d^0 .. d^64
  float cum[C], step[C];                 // SSD: c_i in units of log2(e), d_i
};

// What the two rules take beside q, k and v.
struct LightArgs {
  const float* decay;   // fixed: [heads]
  const bf16* dt;       // SSD: raw step sizes [heads], rows of stride lddt
  long long lddt;
  const float *a_log, *dt_bias, *skip;  // SSD: [heads]
  int groups;
};

__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const float ah = bf16_round(a), bh = bf16_round(b);
  hi = pack2(ah, bh);
  lo = pack2(a - ah, b - bh);
}

template <int DK, bool SSD>
__global__ void __launch_bounds__(256, 1) lightning_chunk_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k, const bf16* __restrict__ v, long long ld, const LightArgs args,
                                                                 float* __restrict__ state, bf16* __restrict__ out, const int* __restrict__ q_indptr, const int* __restrict__ slots, int heads,
                                                                 int dk, int dv, int col_blocks, int min_len) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  LightSmem<DK>& sm = *reinterpret_cast<LightSmem<DK>*>(smem_raw);
  constexpr int LDK = LightSmem<DK>::LDK;
  constexpr int MT = DK / 128 > 0 ? DK / 128 : 1;  // 16-row state tiles per warp (DK = 64: the upper four warps hold none)
  const int h = blockIdx.x / col_blocks, dv0 = (blockIdx.x % col_blocks) * DVC, b = blockIdx.y;
  const int slot = slots[b], q0 = q_indptr[b], q1 = q_indptr[b + 1];
  if (q1 == q0 || q1 - q0 < min_len || slot < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, t4 = lane & 3;
  const int wm = warp & 3, wn = warp >> 2;  // 16 tokens x 32 value columns of the output
  const int ncol = min(DVC, dv - dv0);
  const int kh = SSD ? h * args.groups / heads : h;
  constexpr float L2E = 1.4426950408889634f;
  float rate = 0.f, dt_b = 0.f, skip = 0.f, raw = 0.f;
  if (SSD) {
    rate = -__expf(args.a_log[h]) * L2E, dt_b = args.dt_bias[h], skip = args.skip[h];
    if (tid < C && q0 + tid < q1) raw = __bfloat162float(args.dt[(long long)(q0 + tid) * args.lddt + h]);
  } else {
    const float d = args.decay[h];
    if (tid <= C) sm.pw[tid] = tid == 0 ? 1.f : (d > 0.f ? exp2f((float)tid * log2f(d)) : 0.f);
  }

  float* S = state + (((long long)slot * heads + h) * dk) * dv + dv0;
  float sacc[MT][8][4];
  auto state_row = [&](int m) { return (warp * MT + m) * 16 + gq; };
  const bool has_state = warp * MT * 16 < DK;
  auto store_operand = [&]() {
    if (!has_state) return;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        const int col = n * 8 + 2 * t4, r = state_row(m);
        uint32_t hi, lo;
        split2(sacc[m][n][0], sacc[m][n][1], hi, lo);
        *reinterpret_cast<uint32_t*>(&sm.s_hi[r * LDV + col]) = hi;
        *reinterpret_cast<uint32_t*>(&sm.s_lo[r * LDV + col]) = lo;
        split2(sacc[m][n][2], sacc[m][n][3], hi, lo);
        *reinterpret_cast<uint32_t*>(&sm.s_hi[(r + 8) * LDV + col]) = hi;
        *reinterpret_cast<uint32_t*>(&sm.s_lo[(r + 8) * LDV + col]) = lo;
      }
  };
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int col = n * 8 + 2 * t4;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = state_row(m) + (e >> 1) * 8, c = col + (e & 1);
        sacc[m][n][e] = has_state && r < dk && c < ncol ? S[(long long)r * dv + c] : 0.f;
      }
    }
  store_operand();

  auto stage = [&](int t0, int buf) {
    const int nt = min(C, q1 - t0);
#pragma unroll
    for (int i = 0; i < C * (DK / 8) / 256; ++i) {
      const int c = tid + 256 * i, r = c / (DK / 8), ch = c % (DK / 8);
      const bool ok = r < nt && ch * 8 < dk;
      const long long at = (long long)(t0 + (r < nt ? r : 0)) * ld + (long long)kh * dk + (ok ? ch * 8 : 0);
      cp_async16(&sm.q[buf][r * LDK + ch * 8], q + at, ok);
      cp_async16(&sm.k[buf][r * LDK + ch * 8], k + at, ok);
    }
#pragma unroll
    for (int i = 0; i < C * (DVC / 8) / 256; ++i) {
      const int c = tid + 256 * i, r = c / (DVC / 8), ch = c % (DVC / 8);
      const bool ok = r < nt && ch * 8 < ncol;
      cp_async16(&sm.v[buf][r * LDV + ch * 8], v + (long long)(t0 + (r < nt ? r : 0)) * ld + (long long)h * dv + dv0 + (ok ? ch * 8 : 0), ok);
    }
    cp_async_commit();
  };
  auto silu8 = [](bf16* p, float* f) {
    unpack8(*reinterpret_cast<const bf16x8*>(p), f);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = __fdividef(f[e], 1.f + __expf(-f[e]));
    const bf16x8 r = pack8(f);
    *reinterpret_cast<bf16x8*>(p) = r;
    unpack8(r, f);
  };

  stage(q0, 0);
  int buf = 0;
  for (int t0 = q0; t0 < q1; t0 += C, buf ^= 1) {
    const int nt = min(C, q1 - t0);
    cp_async_wait_all();
    __syncthreads();  // the chunk's rows are here; the other buffer has been read out
    if (t0 + C < q1) stage(t0 + C, buf ^ 1);
    if (SSD) {
      if (warp < 2) {  // step sizes and their running sum, 32 tokens per warp
        const float z = raw + dt_b, s = tid < nt ? (z > 20.f ? z : log1pf(__expf(z))) : 0.f;  // rows past the end leave the state as it is
        float c = s * rate;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float up = __shfl_up_sync(0xffffffffu, c, o);
          if (lane >= o) c += up;
        }
        sm.step[tid] = s;
        sm.cum[tid] = c;
        if (t0 + C + tid < q1) raw = __bfloat162float(args.dt[(long long)(t0 + C + tid) * args.lddt + h]);
      }
      __syncthreads();
      if (warp == 1) sm.cum[tid] += sm.cum[31];
      __syncthreads();
    }
    {  // SiLU in place (zero rows stay zero), and the decayed values
      float f[8];
      if (!SSD) {
#pragma unroll
        for (int i = 0; i < C * (DK / 8) / 256; ++i) {
          const int c = tid + 256 * i, r = c / (DK / 8), ch = c % (DK / 8);
          silu8(&sm.q[buf][r * LDK + ch * 8], f);
          silu8(&sm.k[buf][r * LDK + ch * 8], f);
        }
      }
#pragma unroll
      for (int i = 0; i < C * (DVC / 8) / 256; ++i) {
        const int c = tid + 256 * i, r = c / (DVC / 8), ch = c % (DVC / 8);
        if (SSD)
          unpack8(*reinterpret_cast<const bf16x8*>(&sm.v[buf][r * LDV + ch * 8]), f);
        else
          silu8(&sm.v[buf][r * LDV + ch * 8], f);
        const float w = SSD ? exp2f(sm.cum[C - 1] - sm.cum[r]) * sm.step[r] : r < nt ? sm.pw[nt - 1 - r] : 0.f;
#pragma unroll
        for (int e = 0; e < 8; e += 2) {
          uint32_t hi, lo;
          split2(f[e] * w, f[e + 1] * w, hi, lo);
          *reinterpret_cast<uint32_t*>(&sm.vd_hi[r * LDV + ch * 8 + e]) = hi;
          *reinterpret_cast<uint32_t*>(&sm.vd_lo[r * LDV + ch * 8 + e]) = lo;
        }
      }
    }
    __syncthreads();
    const bf16 *sq = sm.q[buf], *sk = sm.k[buf], *sv = sm.v[buf];

    // ---- O = diag(d^(i+1)) Q S0 and P = decayed Q K^T in one walk over the key width ------------------
    float o[4][4], p[8][4];
#pragma unroll
    for (int n = 0; n < 4; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
#pragma unroll
    for (int n = 0; n < 8; ++n) p[n][0] = p[n][1] = p[n][2] = p[n][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      uint32_t a[4], bb[4];
      frag_a(sq, LDK, wm * 16, ks * 16, lane, a);
#pragma unroll
      for (int n2 = 0; n2 < 2; ++n2) {
        frag_b_kn(sm.s_hi, LDV, ks * 16, wn * 32 + n2 * 16, lane, bb);
        mma16816(o[2 * n2], a, bb[0], bb[1]);
        mma16816(o[2 * n2 + 1], a, bb[2], bb[3]);
        frag_b_kn(sm.s_lo, LDV, ks * 16, wn * 32 + n2 * 16, lane, bb);
        mma16816(o[2 * n2], a, bb[0], bb[1]);
        mma16816(o[2 * n2 + 1], a, bb[2], bb[3]);
      }
#pragma unroll
      for (int n2 = 0; n2 < 4; ++n2) {
        if (n2 <= wm) {  // keys 16 n2 .. 16 n2 + 15: nothing above the diagonal tile
          frag_b_nk(sk, LDK, n2 * 16, ks * 16, lane, bb);
          mma16816(p[2 * n2], a, bb[0], bb[1]);
          mma16816(p[2 * n2 + 1], a, bb[2], bb[3]);
        }
      }
    }
    {
      const float lo = SSD ? exp2f(sm.cum[wm * 16 + gq]) : sm.pw[wm * 16 + gq + 1], hi = SSD ? exp2f(sm.cum[wm * 16 + gq + 8]) : sm.pw[wm * 16 + gq + 9];
#pragma unroll
      for (int n = 0; n < 4; ++n) o[n][0] *= lo, o[n][1] *= lo, o[n][2] *= hi, o[n][3] *= hi;
    }
    // ---- O += P V, P straight from its accumulators ---------------------------------------------------
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      if (ks <= wm) {
        uint32_t ph[4], pl[4], bb[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          float x[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = wm * 16 + gq + (e >> 1) * 8, j = ks * 16 + half * 8 + 2 * t4 + (e & 1);
            if (SSD)
              x[e] = j <= i ? fmaf(p[2 * ks + half][e], exp2f(sm.cum[i] - sm.cum[j]) * sm.step[j], j == i ? skip : 0.f) : 0.f;
            else
              x[e] = j <= i ? p[2 * ks + half][e] * sm.pw[i - j] : 0.f;
          }
          split2(x[0], x[1], ph[2 * half], pl[2 * half]);
          split2(x[2], x[3], ph[2 * half + 1], pl[2 * half + 1]);
        }
#pragma unroll
        for (int n2 = 0; n2 < 2; ++n2) {
          frag_b_kn(sv, LDV, ks * 16, wn * 32 + n2 * 16, lane, bb);
          mma16816(o[2 * n2], ph, bb[0], bb[1]);
          mma16816(o[2 * n2 + 1], ph, bb[2], bb[3]);
          mma16816(o[2 * n2], pl, bb[0], bb[1]);
          mma16816(o[2 * n2 + 1], pl, bb[2], bb[3]);
        }
      }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int c = wn * 32 + n * 8 + 2 * t4, r = wm * 16 + gq;
      if (c < ncol) {
        if (r < nt) *reinterpret_cast<uint32_t*>(out + ((long long)(t0 + r) * heads + h) * dv + dv0 + c) = pack2(o[n][0], o[n][1]);
        if (r + 8 < nt) *reinterpret_cast<uint32_t*>(out + ((long long)(t0 + r + 8) * heads + h) * dv + dv0 + c) = pack2(o[n][2], o[n][3]);
      }
    }
    // ---- S <- d^n S + K^T (decayed V) ------------------------------------------------------------------
    if (has_state) {
      const float dn = SSD ? exp2f(sm.cum[C - 1]) : sm.pw[nt];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) sacc[m][n][e] *= dn;
#pragma unroll
        for (int ks = 0; ks < C / 16; ++ks) {
          uint32_t a[4], bb[4];
          frag_a_t(sk, LDK, (warp * MT + m) * 16, ks * 16, lane, a);
#pragma unroll
          for (int n2 = 0; n2 < 4; ++n2) {
            frag_b_kn(sm.vd_hi, LDV, ks * 16, n2 * 16, lane, bb);
            mma16816(sacc[m][2 * n2], a, bb[0], bb[1]);
            mma16816(sacc[m][2 * n2 + 1], a, bb[2], bb[3]);
            frag_b_kn(sm.vd_lo, LDV, ks * 16, n2 * 16, lane, bb);
            mma16816(sacc[m][2 * n2], a, bb[0], bb[1]);
            mma16816(sacc[m][2 * n2 + 1], a, bb[2], bb[3]);
          }
        }
      }
    }
    __syncthreads();  // every warp has read the old state operand
    if (t0 + C < q1) store_operand();
    // the next chunk's first barrier orders these writes before they are read
  }
  if (has_state) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = state_row(m) + (e >> 1) * 8, c = n * 8 + 2 * t4 + (e & 1);
          if (r < dk && c < ncol) S[(long long)r * dv + c] = sacc[m][n][e];
        }
  }
}

template <int DK, bool SSD>
int launch_lightning(const void* q, const void* k, const void* v, long long ld, const LightArgs& args, void* state, void* out, const void* q_indptr, const void* slots, int num_seqs, int heads,
                     int dk, int dv, int min_len, cudaStream_t stream) {
  static bool set = false;
  if (!set) {
    PG_CUDA(cudaFuncSetAttribute(lightning_chunk_kernel<DK, SSD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(LightSmem<DK>)));
    set = true;
  }
  const int cb = (dv + DVC - 1) / DVC;
  lightning_chunk_kernel<DK, SSD><<<dim3(heads * cb, num_seqs), 256, sizeof(LightSmem<DK>), stream>>>((const bf16*)q, (const bf16*)k, (const bf16*)v, ld, args, (float*)state,
                                                                                                 (bf16*)out, (const int*)q_indptr, (const int*)slots, heads, dk, dv, cb, min_len);
  PG_LAUNCH_CHECK();
  return PG_OK;
}

}  // namespace

extern "C" int pg_lightning_chunked(const void* q, const void* k, const void* v, long long ld, const void* decay, void* state, void* out, const void* q_indptr, const void* slots, int num_seqs,
                                    int heads, int dk, int dv, int min_len, cudaStream_t stream) {
  PG_REQUIRE(dk % 8 == 0 && dk <= 128 && dv % 8 == 0, "lightning_chunked: key width %d (a multiple of 8 up to 128), value width %d (a multiple of 8)", dk, dv);
  PG_REQUIRE(ld % 8 == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)out) & 15) == 0, "lightning_chunked: rows must be 16-byte aligned");
  PG_REQUIRE(num_seqs <= 65535, "lightning_chunked: %d sequences", num_seqs);
  if (num_seqs == 0) return PG_OK;
  LightArgs a = {};
  a.decay = (const float*)decay;
  if (dk <= 64) return launch_lightning<64, false>(q, k, v, ld, a, state, out, q_indptr, slots, num_seqs, heads, dk, dv, min_len, stream);
  return launch_lightning<128, false>(q, k, v, ld, a, state, out, q_indptr, slots, num_seqs, heads, dk, dv, min_len, stream);
}

// State-space duality (operands as in pg_ssd_recurrent, bf16) for the sequences of at least min_len tokens.
extern "C" int pg_ssd_chunked(const void* C_, const void* B, const void* x, long long ld, const void* dt, long long lddt, const void* a_log, const void* dt_bias, const void* D, void* state, void* out,
                              const void* q_indptr, const void* slots, int num_seqs, int heads, int groups, int n, int dv, int min_len, cudaStream_t stream) {
  PG_REQUIRE(n % 8 == 0 && n <= 128 && dv % 8 == 0 && heads % groups == 0, "ssd_chunked: state width %d (a multiple of 8 up to 128), value width %d (a multiple of 8), heads %d / %d", n, dv, heads, groups);
  PG_REQUIRE(ld % 8 == 0 && (((uintptr_t)C_ | (uintptr_t)B | (uintptr_t)x | (uintptr_t)out) & 15) == 0, "ssd_chunked: rows must be 16-byte aligned");
  PG_REQUIRE(num_seqs <= 65535, "ssd_chunked: %d sequences", num_seqs);
  if (num_seqs == 0) return PG_OK;
  const LightArgs a = {nullptr, (const bf16*)dt, lddt, (const float*)a_log, (const float*)dt_bias, (const float*)D, groups};
  if (n <= 64) return launch_lightning<64, true>(C_, B, x, ld, a, state, out, q_indptr, slots, num_seqs, heads, n, dv, min_len, stream);
  return launch_lightning<128, true>(C_, B, x, ld, a, state, out, q_indptr, slots, num_seqs, heads, n, dv, min_len, stream);
}
