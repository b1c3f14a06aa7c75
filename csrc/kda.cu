// Kernels of the KDA + latent-MoE model line (Kimi-K3 shape).
//
//  * kda_recurrent: the delta rule with a decay per key channel.  Per token and head,
//      dec[d] = exp(lower * sigmoid(exp(A_log[h]) * (f[d] + dt_bias[h, d])))   (lower < 0, so dec in (e^lower, 1))
//      S      = S * dec (rows of S[Dk, Dv] scaled)        kv = S^T k
//      S     += k (x) ((v - kv) * sigmoid(b))             out = S^T q
//    with q and k L2-normalised (q also times Dk^-0.5).  The gate arithmetic runs inside the kernel, so the
//    step needs no separate gate launch.  The state layout and the thread mapping are those of the scalar-decay
//    rule in gdn.cu: a CTA takes 32 columns of one (sequence, head), four lanes share a column and each keeps a
//    quarter of its Dk elements in registers; a stage of 8 tokens is normalised into shared memory, then
//    walked in order.  A decode step is one pass over the state (read + write).
//    The same kernel runs two more rules (RULE below): the decay in its softplus form, exp(-exp(A_log) softplus(f + dt_bias)),
//    with query / key heads shared by several value heads, plain linear attention with one fixed decay per head
//    (S = decay S + k (x) v, out = S^T q, SiLU on q, k and v), and linear attention with a decay per token and key channel and a
//    bonus for the current token (out = (S + diag(u) k (x) v)^T q in front of S = diag(dec) S + k (x) v, dec = exp(-exp(f + w0))), and
//    state-space duality, one decay per token and head (d = softplus(f + dt_bias), S = exp(-exp(A_log) d) S + d k (x) v, out = S^T q +
//    D v, keys and queries shared by a group of heads).
//    Those take bf16 or f32 rows and any key width up to 256.
//  * attnres_mix: the attention-residual mix.  Every token keeps up to `cap` snapshot rows of its own residual
//    stream; a mix scores each of the first nb snapshots and the current row with
//    dot(x / rms(x), score_w) and returns the softmax-weighted sum of the un-normalised rows.
//
// Functional parity with pegainfer-k3/kernels/tilelang_defs.py:67-139 (attnres_scores / attnres_mix) and
// :304-410 (kda_core) and pegainfer-kernels/csrc/k3/k3_flash_kda.cu (chunked prefill of the same rule).
#include "api.h"
#include "common.cuh"
#include "types.cuh"

namespace {

constexpr int KDA_STAGE = 8;
constexpr int KDA_COLS = 32;

// What a token does to the state.  BOUNDED and SOFTPLUS are the delta rule with a decay per key channel and two forms of
// the decay; DECAY is linear attention with a fixed decay per head (no correction term), WKV with a decay per token and key
// channel, read in front of the update with a bonus for the current token, SSD with a decay and a step size per token and head.
enum { RULE_BOUNDED = 0, RULE_SOFTPLUS = 1, RULE_DECAY = 2, RULE_WKV = 3, RULE_SSD = 4 };

template <typename T>
struct RecArgs {
  const T *q, *k, *v;  // token rows of stride ld; q and k [kv_heads * dk], v [heads * dv]
  long long ld;
  const void* f;  // raw decay projection [heads * dk]: T (BOUNDED) or f32 (SOFTPLUS, WKV); SSD: raw step sizes T [heads]
  long long ldf;
  const T* b;  // raw step-size projection [heads]
  long long ldb;
  const float *a_log, *dt_bias, *decay;  // decay [heads]: DECAY; WKV: dt_bias = w0 [heads * dk], decay = the bonus u [heads * dk]; SSD: dt_bias [heads], decay = D [heads]
  float lower;
  float* state;
  T* out;
  const int *q_indptr, *slots;
  int heads, kv_heads, dk, dv, col_groups;
  int skip_len;  // > 0: sequences of at least that many tokens belong to another kernel
};

// XW = false: four adjacent lanes share a state column and reduce with shuffles (prompt chunks: no barrier per token).
// XW = true: a warp owns one quarter of Dk for all 32 columns, so every state load and store of a warp is one 128-byte row
// and the shared-memory reads of k, q and the decays are broadcasts; the four quarters meet through shared memory with two
// barriers per token (decode rows and other steps of a few tokens).
// DK is the key width rounded up to an instantiated size; entries past dk are zero (PAD).
template <typename T, int DK, bool XW, int RULE, bool PAD>
__global__ void __launch_bounds__(128) kda_recurrent_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long long ld, const void* __restrict__ f, long long ldf,
                                                            const T* __restrict__ b, long long ldb, const float* __restrict__ a_log, const float* __restrict__ dt_bias, const float* __restrict__ decay,
                                                            float lower, float* __restrict__ state, T* __restrict__ out, const int* __restrict__ q_indptr, const int* __restrict__ slots, int heads,
                                                            int kv_heads, int dk_arg, int dv, int col_groups, int skip_len) {
  constexpr int QK = DK / 4;   // state elements per thread
  constexpr int QS = QK + 4;   // padded quarter stride: the four quarters land in different banks
  constexpr int QL = DK / 32;  // elements per lane when a warp holds one token
  constexpr bool DELTA = RULE == RULE_BOUNDED || RULE == RULE_SOFTPLUS;
  constexpr bool KEYED = RULE != RULE_DECAY && RULE != RULE_SSD;  // a decay per key channel
  __shared__ __align__(16) float sq[KDA_STAGE][4 * QS], sk[KDA_STAGE][4 * QS], sd[KEYED ? KDA_STAGE : 1][4 * QS];
  __shared__ float sv[KDA_STAGE][KDA_COLS], sb[KDA_STAGE], se[RULE == RULE_SSD ? KDA_STAGE : 1];
  __shared__ float red_kv[4][KDA_COLS], red_o[DELTA ? 1 : 2][4][KDA_COLS];
  const int dk = PAD ? dk_arg : DK;
  const int h = blockIdx.x / col_groups, cg = blockIdx.x % col_groups, seq = blockIdx.y;
  const int slot = slots[seq];
  const int q0 = q_indptr[seq], q1 = q_indptr[seq + 1];
  if (q1 == q0 || slot < 0) return;
  if (RULE != RULE_BOUNDED && skip_len > 0 && q1 - q0 >= skip_len) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qtr = XW ? warp : (tid & 3), lc = XW ? lane : (tid >> 2), col = cg * KDA_COLS + lc;
  const bool owner = col < dv;
  float* S = state + (((long long)slot * heads + h) * dk) * dv;  // [dk][dv], v contiguous
  // Shuffle mapping: a thread's own elements sit DK / 4 rows apart, so a warp reads 32-byte pieces of four rows.  Staging
  // the CTA's slice through shared memory instead was measured slower (200 us against 111 us for 32 decode rows of 96
  // heads: the extra 17 KB per CTA costs resident CTAs); the XW mapping reads whole rows without it (86 us).
  float s_col[QK];
#pragma unroll
  for (int i = 0; i < QK; ++i) s_col[i] = owner && (!PAD || qtr * QK + i < dk) ? S[(long long)(qtr * QK + i) * dv + col] : 0.f;
  const int kh = RULE == RULE_SOFTPLUS || RULE == RULE_SSD ? h * kv_heads / heads : h;
  const float q_scale = DELTA ? rsqrtf((float)dk) : 1.f;
  const float a = DELTA || RULE == RULE_SSD ? __expf(a_log[h]) : 0.f;
  const float fixed = RULE == RULE_DECAY || RULE == RULE_SSD ? decay[h] : 0.f;

  for (int t0 = q0; t0 < q1; t0 += KDA_STAGE) {
    const int nt = min(KDA_STAGE, q1 - t0);
    // stage: each warp prepares two tokens' q and k (unit rows, or SiLU of the projections) and their decays
    for (int j = warp; j < nt; j += 4) {
      const long long row = (long long)(t0 + j);
      const T* qp = q + row * ld + (long long)kh * dk;
      const T* kp = k + row * ld + (long long)kh * dk;
      float rq[QL], rk[QL], qs = 0.f, ks = 0.f;
#pragma unroll
      for (int i = 0; i < QL; ++i) {
        const bool in = !PAD || lane + 32 * i < dk;
        rq[i] = in ? to_f32(qp[lane + 32 * i]) : 0.f;
        rk[i] = in ? to_f32(kp[lane + 32 * i]) : 0.f;
        if (DELTA) {
          qs += rq[i] * rq[i];
          ks += rk[i] * rk[i];
        } else if (RULE == RULE_WKV) {
          if (in) qs += rq[i] * rk[i] * decay[h * dk + lane + 32 * i];
        } else if (RULE == RULE_DECAY) {  // the activation's result is what the layer works with, in the activation type
          rq[i] = to_f32(from_f32<T>(rq[i] / (1.f + __expf(-rq[i]))));
          rk[i] = to_f32(from_f32<T>(rk[i] / (1.f + __expf(-rk[i]))));
        }
      }
      float qn = 1.f, kn = 1.f;
      if (DELTA) {
        qs = warp_sum(qs);
        ks = warp_sum(ks);
        qn = rsqrtf(qs + 1e-6f) * q_scale, kn = rsqrtf(ks + 1e-6f);
      }
      if (RULE == RULE_WKV) {  // what the token's own value counts
        qs = warp_sum(qs);
        if (lane == 0) sb[j] = qs;
      }
#pragma unroll
      for (int i = 0; i < QL; ++i) {
        const int e = lane + 32 * i, at = (e / QK) * QS + (e % QK);
        sq[j][at] = rq[i] * qn;
        sk[j][at] = rk[i] * kn;
        if (RULE == RULE_BOUNDED) {
          const float raw = to_f32(((const T*)f)[row * ldf + (long long)h * dk + e]) + dt_bias[h * dk + e];
          sd[j][at] = __expf(lower / (1.f + __expf(-a * raw)));
        } else if (RULE == RULE_SOFTPLUS) {
          float dec = 1.f;
          if (!PAD || e < dk) {
            const float raw = ((const float*)f)[row * ldf + (long long)h * dk + e] + dt_bias[h * dk + e];
            dec = __expf(-a * (raw > 20.f ? raw : log1pf(__expf(raw))));
          }
          sd[j][at] = dec;
        } else if (RULE == RULE_WKV) {
          sd[j][at] = !PAD || e < dk ? __expf(-__expf(((const float*)f)[row * ldf + (long long)h * dk + e] + dt_bias[h * dk + e])) : 1.f;
        }
      }
    }
    for (int idx = tid; idx < nt * KDA_COLS; idx += 128) {
      const int j = idx / KDA_COLS, d = cg * KDA_COLS + idx % KDA_COLS;
      float x = d < dv ? to_f32(v[(long long)(t0 + j) * ld + (long long)h * dv + d]) : 0.f;
      if (RULE == RULE_DECAY) x = to_f32(from_f32<T>(x / (1.f + __expf(-x))));
      sv[j][idx % KDA_COLS] = x;
    }
    if (RULE == RULE_SSD && tid < nt) {
      const float raw = to_f32(((const T*)f)[(long long)(t0 + tid) * ldf + h]) + dt_bias[h], d = raw > 20.f ? raw : log1pf(__expf(raw));
      sb[tid] = d;
      se[tid] = __expf(-a * d);
    }
    if (DELTA && tid < nt) sb[tid] = 1.f / (1.f + __expf(-to_f32(b[(long long)(t0 + tid) * ldb + h])));
    __syncthreads();
    for (int j = 0; j < nt; ++j) {
      const float4* kq = reinterpret_cast<const float4*>(&sk[j][qtr * QS]);
      const float4* qq = reinterpret_cast<const float4*>(&sq[j][qtr * QS]);
      float delta = RULE == RULE_SSD ? sv[j][lc] * sb[j] : sv[j][lc];
      if (DELTA) {
        const float4* dq = reinterpret_cast<const float4*>(&sd[DELTA ? j : 0][qtr * QS]);
        float4 kv4 = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < QK / 4; ++i) {
          const float4 kk = kq[i], dd = dq[i];
          s_col[4 * i + 0] *= dd.x;
          s_col[4 * i + 1] *= dd.y;
          s_col[4 * i + 2] *= dd.z;
          s_col[4 * i + 3] *= dd.w;
          kv4.x += s_col[4 * i + 0] * kk.x;
          kv4.y += s_col[4 * i + 1] * kk.y;
          kv4.z += s_col[4 * i + 2] * kk.z;
          kv4.w += s_col[4 * i + 3] * kk.w;
        }
        float kv = (kv4.x + kv4.y) + (kv4.z + kv4.w);
        if (XW) {
          red_kv[qtr][lc] = kv;
          __syncthreads();
          kv = (red_kv[0][lc] + red_kv[1][lc]) + (red_kv[2][lc] + red_kv[3][lc]);
        } else {
          kv += __shfl_xor_sync(0xffffffffu, kv, 1);
          kv += __shfl_xor_sync(0xffffffffu, kv, 2);
        }
        delta = (delta - kv) * sb[j];
      }
      float4 o4 = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < QK / 4; ++i) {
        const float4 kk = kq[i], qv = qq[i];
        if (RULE == RULE_WKV) {
          const float4 dd = reinterpret_cast<const float4*>(&sd[KEYED ? j : 0][qtr * QS])[i];
          o4.x += s_col[4 * i + 0] * qv.x;
          o4.y += s_col[4 * i + 1] * qv.y;
          o4.z += s_col[4 * i + 2] * qv.z;
          o4.w += s_col[4 * i + 3] * qv.w;
          s_col[4 * i + 0] = s_col[4 * i + 0] * dd.x + kk.x * delta;
          s_col[4 * i + 1] = s_col[4 * i + 1] * dd.y + kk.y * delta;
          s_col[4 * i + 2] = s_col[4 * i + 2] * dd.z + kk.z * delta;
          s_col[4 * i + 3] = s_col[4 * i + 3] * dd.w + kk.w * delta;
          continue;
        }
        if (!DELTA) {
          const float dec = RULE == RULE_SSD ? se[RULE == RULE_SSD ? j : 0] : fixed;
          s_col[4 * i + 0] *= dec;
          s_col[4 * i + 1] *= dec;
          s_col[4 * i + 2] *= dec;
          s_col[4 * i + 3] *= dec;
        }
        s_col[4 * i + 0] += kk.x * delta;
        s_col[4 * i + 1] += kk.y * delta;
        s_col[4 * i + 2] += kk.z * delta;
        s_col[4 * i + 3] += kk.w * delta;
        o4.x += s_col[4 * i + 0] * qv.x;
        o4.y += s_col[4 * i + 1] * qv.y;
        o4.z += s_col[4 * i + 2] * qv.z;
        o4.w += s_col[4 * i + 3] * qv.w;
      }
      float o = (o4.x + o4.y) + (o4.z + o4.w);
      if (XW) {
        // two buffers: with the delta rule the barrier in front of it orders a token's reads before the next token's
        // writes, without it the next token writes the other buffer and the one after that comes behind its barrier
        red_o[DELTA ? 0 : j & 1][qtr][lc] = o;
        __syncthreads();  // also orders this token's reads of red_kv before the next token's writes
        o = (red_o[DELTA ? 0 : j & 1][0][lc] + red_o[DELTA ? 0 : j & 1][1][lc]) + (red_o[DELTA ? 0 : j & 1][2][lc] + red_o[DELTA ? 0 : j & 1][3][lc]);
      } else {
        o += __shfl_xor_sync(0xffffffffu, o, 1);
        o += __shfl_xor_sync(0xffffffffu, o, 2);
      }
      if (RULE == RULE_WKV) o += sb[j] * delta;
      if (RULE == RULE_SSD) o += fixed * sv[j][lc];
      if (owner && qtr == 0) out[((long long)(t0 + j) * heads + h) * dv + col] = from_f32<T>(o);
    }
    __syncthreads();
  }
  if (owner) {
#pragma unroll
    for (int i = 0; i < QK; ++i)
      if (!PAD || qtr * QK + i < dk) S[(long long)(qtr * QK + i) * dv + col] = s_col[i];
  }
}

template <typename T, int DK, int RULE, bool PAD>
cudaError_t launch_rule(const RecArgs<T>& p, dim3 grid, bool few, cudaStream_t stream) {
  auto kernel = few ? kda_recurrent_kernel<T, DK, true, RULE, PAD> : kda_recurrent_kernel<T, DK, false, RULE, PAD>;
  // launched in plain stream order: a successor that starts early holds CTA slots of this kernel's long-running blocks
  // (prompt of 2048 tokens: 2.5 ms with programmatic launch, 2.1 ms without)
  kernel<<<grid, 128, 0, stream>>>(p.q, p.k, p.v, p.ld, p.f, p.ldf, p.b, p.ldb, p.a_log, p.dt_bias, p.decay, p.lower, p.state, p.out, p.q_indptr, p.slots, p.heads, p.kv_heads, p.dk, p.dv, p.col_groups,
                                   p.skip_len);
  return cudaSuccess;
}
// any key width up to 256, on the next larger instantiated size
template <typename T, int RULE>
cudaError_t launch_padded(const RecArgs<T>& p, dim3 grid, bool few, cudaStream_t stream) {
  if (p.dk == 128) return launch_rule<T, 128, RULE, false>(p, grid, few, stream);
  if (p.dk == 64) return launch_rule<T, 64, RULE, false>(p, grid, few, stream);
  if (p.dk <= 32) return launch_rule<T, 32, RULE, true>(p, grid, few, stream);
  if (p.dk <= 64) return launch_rule<T, 64, RULE, true>(p, grid, few, stream);
  if (p.dk <= 128) return launch_rule<T, 128, RULE, true>(p, grid, few, stream);
  return launch_rule<T, 256, RULE, true>(p, grid, few, stream);
}

template <typename T>
int run_rule(int rule, RecArgs<T> p, int num_seqs, int max_q_len, cudaStream_t stream) {
  p.col_groups = (p.dv + KDA_COLS - 1) / KDA_COLS;
  const dim3 grid(p.heads * p.col_groups, num_seqs);
  const bool few = max_q_len <= 4;  // decode rows and verify steps: the row-coalesced mapping
  PG_CUDA(rule == RULE_SOFTPLUS ? (launch_padded<T, RULE_SOFTPLUS>(p, grid, few, stream))
          : rule == RULE_WKV    ? (launch_padded<T, RULE_WKV>(p, grid, few, stream))
          : rule == RULE_SSD    ? (launch_padded<T, RULE_SSD>(p, grid, few, stream))
                                : (launch_padded<T, RULE_DECAY>(p, grid, few, stream)));
  PG_LAUNCH_CHECK();
  return PG_OK;
}

constexpr int ATTNRES_MAX = 16;  // candidates of one mix (snapshots + the current row)

// One CTA of 256 threads per token.  Pass 1: sum of squares and dot with score_w for every candidate; pass 2: softmax of
// the scores and the weighted sum (the rows come back from L1 / L2).
__global__ void __launch_bounds__(256) attnres_mix_kernel(const bf16* __restrict__ cur, long long ld_cur, const bf16* __restrict__ snaps, long long ld_tok,
                                                           const float* __restrict__ score_w, bf16* __restrict__ out, long long ld_out, int nb, int hidden,
                                                           float eps) {
  PG_PDL_ENTRY();
  __shared__ float red[2][ATTNRES_MAX][8];
  __shared__ float prob[ATTNRES_MAX];
  const long long t = blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nvec = hidden / 8;
  const int nc = nb + 1;
  auto row = [&](int c) { return c < nb ? snaps + t * ld_tok + (long long)c * hidden : cur + t * ld_cur; };
  for (int c = 0; c < nc; ++c) {
    const bf16x8* xr = reinterpret_cast<const bf16x8*>(row(c));
    float ss = 0.f, dot = 0.f;
    for (int i = tid; i < nvec; i += 256) {
      float x[8];
      unpack8(xr[i], x);
      const float4 w0 = reinterpret_cast<const float4*>(score_w)[2 * i], w1 = reinterpret_cast<const float4*>(score_w)[2 * i + 1];
      ss += x[0] * x[0] + x[1] * x[1] + x[2] * x[2] + x[3] * x[3] + x[4] * x[4] + x[5] * x[5] + x[6] * x[6] + x[7] * x[7];
      dot += x[0] * w0.x + x[1] * w0.y + x[2] * w0.z + x[3] * w0.w + x[4] * w1.x + x[5] * w1.y + x[6] * w1.z + x[7] * w1.w;
    }
    ss = warp_sum(ss);
    dot = warp_sum(dot);
    if (lane == 0) red[0][c][warp] = ss, red[1][c][warp] = dot;
  }
  __syncthreads();
  if (tid == 0) {
    float sc[ATTNRES_MAX], mx = -1e30f, den = 0.f;
    for (int c = 0; c < nc; ++c) {
      float ss = 0.f, dot = 0.f;
      for (int w = 0; w < 8; ++w) ss += red[0][c][w], dot += red[1][c][w];
      sc[c] = dot * rsqrtf(ss / (float)hidden + eps);
      mx = fmaxf(mx, sc[c]);
    }
    for (int c = 0; c < nc; ++c) den += (sc[c] = __expf(sc[c] - mx));
    for (int c = 0; c < nc; ++c) prob[c] = sc[c] / den;
  }
  __syncthreads();
  for (int i = tid; i < nvec; i += 256) {
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int c = 0; c < nc; ++c) {
      float x[8];
      unpack8(reinterpret_cast<const bf16x8*>(row(c))[i], x);
      const float p = prob[c];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] += p * x[j];
    }
    reinterpret_cast<bf16x8*>(out + t * ld_out)[i] = pack8(acc);
  }
}

}  // namespace

extern "C" int pg_kda_recurrent(const void* q, const void* k, const void* v, long long ld, const void* f, long long ldf, const void* b, long long ldb,
                                const void* a_log, const void* dt_bias, float lower, void* state, void* out, const void* q_indptr, const void* slots,
                                int num_seqs, int heads, int dk, int dv, int max_q_len, cudaStream_t stream) {
  PG_REQUIRE(dv <= 128 && lower < 0.f, "kda_recurrent: dv=%d must be <= 128 and the decay lower bound %f negative", dv, (double)lower);
  if (num_seqs == 0) return PG_OK;
  RecArgs<bf16> p = {(const bf16*)q, (const bf16*)k, (const bf16*)v, ld, f, ldf, (const bf16*)b, ldb, (const float*)a_log, (const float*)dt_bias, nullptr, lower,
                     (float*)state, (bf16*)out, (const int*)q_indptr, (const int*)slots, heads, heads, dk, dv, (dv + KDA_COLS - 1) / KDA_COLS, 0};
  const dim3 grid(heads * p.col_groups, num_seqs);
  const bool few = max_q_len <= 4;
  if (dk == 128)
    PG_CUDA((launch_rule<bf16, 128, RULE_BOUNDED, false>(p, grid, few, stream)));
  else if (dk == 64)
    PG_CUDA((launch_rule<bf16, 64, RULE_BOUNDED, false>(p, grid, few, stream)));
  else if (dk == 32)
    PG_CUDA((launch_rule<bf16, 32, RULE_BOUNDED, false>(p, grid, few, stream)));
  else {
    pg_set_error("kda_recurrent: dk=%d not supported (32, 64, 128)", dk);
    return PG_ERR_UNSUPPORTED;
  }
  PG_LAUNCH_CHECK();
  return PG_OK;
}

// The delta rule with the decay exp(-exp(A_log) * softplus(f + dt_bias)), f in f32, and query / key heads that several
// value heads may share.
extern "C" int pg_channel_delta(const void* q, const void* k, const void* v, long long ld, const void* f, long long ldf, const void* b, long long ldb, const void* a_log, const void* dt_bias,
                                void* state, void* out, const void* q_indptr, const void* slots, int num_seqs, int heads, int kv_heads, int dk, int dv, int max_q_len, int skip_len, int is_f32,
                                cudaStream_t stream) {
  PG_REQUIRE(dk >= 1 && dk <= 256 && dv >= 1 && heads % kv_heads == 0, "channel_delta: heads %d / %d, key width %d (at most 256), value width %d", heads, kv_heads, dk, dv);
  PG_REQUIRE(num_seqs <= 65535, "channel_delta: %d sequences", num_seqs);
  if (num_seqs == 0) return PG_OK;
  if (is_f32) {
    RecArgs<float> p = {(const float*)q, (const float*)k, (const float*)v, ld, f, ldf, (const float*)b, ldb, (const float*)a_log, (const float*)dt_bias, nullptr, 0.f,
                        (float*)state, (float*)out, (const int*)q_indptr, (const int*)slots, heads, kv_heads, dk, dv, 0, skip_len};
    return run_rule<float>(RULE_SOFTPLUS, p, num_seqs, max_q_len, stream);
  }
  RecArgs<bf16> p = {(const bf16*)q, (const bf16*)k, (const bf16*)v, ld, f, ldf, (const bf16*)b, ldb, (const float*)a_log, (const float*)dt_bias, nullptr, 0.f,
                     (float*)state, (bf16*)out, (const int*)q_indptr, (const int*)slots, heads, kv_heads, dk, dv, 0, skip_len};
  return run_rule<bf16>(RULE_SOFTPLUS, p, num_seqs, max_q_len, stream);
}

// Linear attention with a fixed decay per head: S <- decay S + k v^T, o = S^T q, with SiLU on q, k and v inside.
extern "C" int pg_decay_recurrent(const void* q, const void* k, const void* v, long long ld, const void* decay, void* state, void* out, const void* q_indptr, const void* slots, int num_seqs,
                                  int heads, int dk, int dv, int max_q_len, int skip_len, int is_f32, cudaStream_t stream) {
  PG_REQUIRE(dk >= 1 && dk <= 256 && dv >= 1, "decay_recurrent: key width %d (at most 256), value width %d", dk, dv);
  PG_REQUIRE(num_seqs <= 65535, "decay_recurrent: %d sequences", num_seqs);
  if (num_seqs == 0) return PG_OK;
  if (is_f32) {
    RecArgs<float> p = {(const float*)q, (const float*)k, (const float*)v, ld, nullptr, 0, nullptr, 0, nullptr, nullptr, (const float*)decay, 0.f,
                        (float*)state, (float*)out, (const int*)q_indptr, (const int*)slots, heads, heads, dk, dv, 0, skip_len};
    return run_rule<float>(RULE_DECAY, p, num_seqs, max_q_len, stream);
  }
  RecArgs<bf16> p = {(const bf16*)q, (const bf16*)k, (const bf16*)v, ld, nullptr, 0, nullptr, 0, nullptr, nullptr, (const float*)decay, 0.f,
                     (float*)state, (bf16*)out, (const int*)q_indptr, (const int*)slots, heads, heads, dk, dv, 0, skip_len};
  return run_rule<bf16>(RULE_DECAY, p, num_seqs, max_q_len, stream);
}

// Linear attention with the decay exp(-exp(f + w0)) per token and key channel (f in f32) and the bonus u [heads, dk] for the
// current token: o = (S + diag(u) k v^T)^T r, then S <- diag(decay) S + k v^T.
extern "C" int pg_wkv_recurrent(const void* r, const void* k, const void* v, long long ld, const void* f, long long ldf, const void* w0, const void* u, void* state, void* out, const void* q_indptr,
                                const void* slots, int num_seqs, int heads, int dk, int dv, int max_q_len, int skip_len, int is_f32, cudaStream_t stream) {
  PG_REQUIRE(dk >= 1 && dk <= 256 && dv >= 1, "wkv_recurrent: key width %d (at most 256), value width %d", dk, dv);
  PG_REQUIRE(num_seqs <= 65535, "wkv_recurrent: %d sequences", num_seqs);
  if (num_seqs == 0) return PG_OK;
  if (is_f32) {
    RecArgs<float> p = {(const float*)r, (const float*)k, (const float*)v, ld, f, ldf, nullptr, 0, nullptr, (const float*)w0, (const float*)u, 0.f,
                        (float*)state, (float*)out, (const int*)q_indptr, (const int*)slots, heads, heads, dk, dv, 0, skip_len};
    return run_rule<float>(RULE_WKV, p, num_seqs, max_q_len, stream);
  }
  RecArgs<bf16> p = {(const bf16*)r, (const bf16*)k, (const bf16*)v, ld, f, ldf, nullptr, 0, nullptr, (const float*)w0, (const float*)u, 0.f,
                     (float*)state, (bf16*)out, (const int*)q_indptr, (const int*)slots, heads, heads, dk, dv, 0, skip_len};
  return run_rule<bf16>(RULE_WKV, p, num_seqs, max_q_len, stream);
}

// State-space duality: x [T, heads, dv] rows of stride ld, B and C [T, groups, n] rows of the same stride, dt [T, heads] raw step sizes of
// stride lddt; d = softplus(dt + dt_bias): S <- exp(-exp(a_log) d) S + d B x^T, out = S^T C + D x.
extern "C" int pg_ssd_recurrent(const void* C, const void* B, const void* x, long long ld, const void* dt, long long lddt, const void* a_log, const void* dt_bias, const void* D, void* state, void* out,
                                const void* q_indptr, const void* slots, int num_seqs, int heads, int groups, int n, int dv, int max_q_len, int skip_len, int is_f32, cudaStream_t stream) {
  PG_REQUIRE(n >= 1 && n <= 256 && dv >= 1 && heads % groups == 0, "ssd_recurrent: heads %d / %d, state width %d (at most 256), value width %d", heads, groups, n, dv);
  PG_REQUIRE(num_seqs <= 65535, "ssd_recurrent: %d sequences", num_seqs);
  if (num_seqs == 0) return PG_OK;
  if (is_f32) {
    RecArgs<float> p = {(const float*)C, (const float*)B, (const float*)x, ld, dt, lddt, nullptr, 0, (const float*)a_log, (const float*)dt_bias, (const float*)D, 0.f,
                        (float*)state, (float*)out, (const int*)q_indptr, (const int*)slots, heads, groups, n, dv, 0, skip_len};
    return run_rule<float>(RULE_SSD, p, num_seqs, max_q_len, stream);
  }
  RecArgs<bf16> p = {(const bf16*)C, (const bf16*)B, (const bf16*)x, ld, dt, lddt, nullptr, 0, (const float*)a_log, (const float*)dt_bias, (const float*)D, 0.f,
                     (float*)state, (bf16*)out, (const int*)q_indptr, (const int*)slots, heads, groups, n, dv, 0, skip_len};
  return run_rule<bf16>(RULE_SSD, p, num_seqs, max_q_len, stream);
}

extern "C" int pg_attnres_mix(const void* cur, long long ld_cur, const void* snaps, long long ld_tok, const void* score_w, void* out, long long ld_out,
                              int tokens, int nb, int hidden, float eps, cudaStream_t stream) {
  PG_REQUIRE(nb >= 0 && nb + 1 <= ATTNRES_MAX && hidden % 8 == 0 && ld_cur % 8 == 0 && ld_tok % 8 == 0 && ld_out % 8 == 0,
             "attnres_mix: %d snapshots (at most %d) and a hidden size %d that is a multiple of 8", nb, ATTNRES_MAX - 1, hidden);
  if (tokens == 0) return PG_OK;
  PG_CUDA(launch_pdl(attnres_mix_kernel, dim3(tokens), dim3(256), (size_t)(0), stream, (const bf16*)cur, ld_cur, (const bf16*)snaps, ld_tok,
                     (const float*)score_w, (bf16*)out, ld_out, nb, hidden, eps));
  PG_LAUNCH_CHECK();
  return PG_OK;
}
