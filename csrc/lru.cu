// Gated linear recurrence per channel (the recurrent block of Griffin): with r and i the sigmoids of two block-diagonal
// projections of u,
//   log a = -8 r softplus(lam),   S <- a S + sqrt(1 - a^2) i u,   out = S * gelu_tanh(y + y_bias) * scale,
// everything in 32 bits but u, y and out.  a and 1 - a^2 come from e = exp(log a) - 1, formed without cancellation: a = 1 + e, 1 - a^2 =
// -e (2 + e).
//
//  * gated_lru_scan: prompts.  A CTA owns 32 channels of a sequence; 16 warps take 8 tokens each of a tile of 128.  Every warp runs
//    its tokens from zero and hands the product of its decays and its result to the others; the tile's carry is then walked over
//    the warps in front, and the tokens run again from there (from registers).  The next tile's rows are loaded meanwhile.
//  * gated_lru_few: decode rows and other short steps, a thread per channel.
#include "api.h"
#include "common.cuh"
#include "types.cuh"

namespace {

constexpr int LC = 32;   // channels of a scan CTA
constexpr int LW = 16;   // its warps
constexpr int LT = 8;    // tokens of a warp per tile
constexpr int FEW = 4;   // steps of at most that many tokens per sequence: a thread per channel

template <typename T>
struct LruArgs {
  const float* gates;  // [tokens, blocks, 2 * part] (r | i)
  const float* gate_bias;
  const T* u;
  long long ldu;
  const float* lam;
  const T* y;
  long long ldy;
  const float* y_bias;
  float* state;  // [slots, width]
  T* out;
  long long ldo;
  const int *q_indptr, *slots;
  int width, part;
  float scale;
};

__device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(__expf(x)); }
__device__ __forceinline__ float sigmoidf(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

// decay and input of one token of a channel; k8 = -8 softplus(lam)
__device__ __forceinline__ void gate_pair(float r, float i, float u, float k8, float& a, float& b) {
  const float la = k8 * sigmoidf(r), e = la + exp_tail(la);
  a = 1.f + e;
  b = sqrtf(-e * (2.f + e)) * sigmoidf(i) * u;
}

template <typename T>
__global__ void __launch_bounds__(LW * 32) gated_lru_scan_kernel(const LruArgs<T> p) {
  PG_PDL_ENTRY();
  __shared__ float sa[2][LW][LC], sb[2][LW][LC];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c = blockIdx.x * LC + lane, seq = blockIdx.y;
  const int slot = p.slots[seq], q0 = p.q_indptr[seq], q1 = p.q_indptr[seq + 1];
  if (q1 == q0 || slot < 0) return;
  const bool in = c < p.width;
  const int cc = in ? c : 0, blk = cc / p.part;
  const long long g_at = (long long)blk * 2 * p.part + cc % p.part, g_ld = 2ll * p.width;
  const float br = p.gate_bias[g_at], bi = p.gate_bias[g_at + p.part], k8 = -8.f * softplus(p.lam[cc]), yb = p.y_bias[cc];
  float S = in ? p.state[(long long)slot * p.width + c] : 0.f;
  float r[LT], i[LT];
  T u[LT], y[LT];
  // byte strides in 32 bits: one widening multiply-add per address
  const int ldg = (int)(g_ld * sizeof(float)), ldu = (int)(p.ldu * sizeof(T)), ldy = (int)(p.ldy * sizeof(T)), ldo = (int)(p.ldo * sizeof(T));
  auto at = [](auto* base, int t, int ld) { return reinterpret_cast<decltype(base)>(reinterpret_cast<uintptr_t>(base) + (long long)t * ld); };
  const float* gp = p.gates + g_at;
  const T *up = p.u + cc, *yp = p.y + cc;
  T* op = p.out + cc;
  auto load = [&](int t0) {  // rows past the end: the last one once more, so that nothing is conditional and all loads are in flight
#pragma unroll
    for (int j = 0; j < LT; ++j) {
      const int t = min(t0 + warp * LT + j, q1 - 1);
      const float* g = at(gp, t, ldg);
      r[j] = g[0], i[j] = g[p.part];
      u[j] = *at(up, t, ldu), y[j] = *at(yp, t, ldy);
    }
  };
  load(q0);
  for (int t0 = q0, buf = 0; t0 < q1; t0 += LW * LT, buf ^= 1) {
    float a[LT], b[LT], g[LT], A = 1.f, B = 0.f;
#pragma unroll
    for (int j = 0; j < LT; ++j) {
      gate_pair(r[j] + br, i[j] + bi, to_f32(u[j]), k8, a[j], b[j]);
      g[j] = glu_act(to_f32(y[j]) + yb, true) * p.scale;
      if (t0 + warp * LT + j >= q1) a[j] = 1.f, b[j] = 0.f;  // rows past the end leave the state as it is
      A *= a[j];
      B = fmaf(a[j], B, b[j]);
    }
    if (t0 + LW * LT < q1) load(t0 + LW * LT);
    sa[buf][warp][lane] = A, sb[buf][warp][lane] = B;
    __syncthreads();
    float mine = S;
#pragma unroll
    for (int w = 0; w < LW; ++w) {
      if (w == warp) mine = S;
      S = fmaf(sa[buf][w][lane], S, sb[buf][w][lane]);
    }
#pragma unroll
    for (int j = 0; j < LT; ++j) {
      const int t = t0 + warp * LT + j;
      mine = fmaf(a[j], mine, b[j]);
      if (in && t < q1) *at(op, t, ldo) = from_f32<T>(mine * g[j]);
    }
  }
  if (in && warp == 0) p.state[(long long)slot * p.width + c] = S;
}

template <typename T>
__global__ void __launch_bounds__(128) gated_lru_few_kernel(const LruArgs<T> p) {
  PG_PDL_ENTRY();
  const int c = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.y;
  const int slot = p.slots[seq], q0 = p.q_indptr[seq], q1 = p.q_indptr[seq + 1];
  if (q1 == q0 || slot < 0 || c >= p.width) return;
  const long long g_at = (long long)(c / p.part) * 2 * p.part + c % p.part, g_ld = 2ll * p.width;
  const float br = p.gate_bias[g_at], bi = p.gate_bias[g_at + p.part], k8 = -8.f * softplus(p.lam[c]), yb = p.y_bias[c];
  float S = p.state[(long long)slot * p.width + c];
  for (long long t = q0; t < q1; ++t) {
    float a, b;
    gate_pair(p.gates[t * g_ld + g_at] + br, p.gates[t * g_ld + g_at + p.part] + bi, to_f32(p.u[t * p.ldu + c]), k8, a, b);
    S = fmaf(a, S, b);
    p.out[t * p.ldo + c] = from_f32<T>(S * glu_act(to_f32(p.y[t * p.ldy + c]) + yb, true) * p.scale);
  }
  p.state[(long long)slot * p.width + c] = S;
}

template <typename T>
int run_lru(const LruArgs<T>& p, int num_seqs, int max_q_len, cudaStream_t stream) {
  if (max_q_len <= FEW)
    PG_CUDA(launch_pdl(gated_lru_few_kernel<T>, dim3((p.width + 127) / 128, num_seqs), dim3(128), (size_t)0, stream, p));
  else
    PG_CUDA(launch_pdl(gated_lru_scan_kernel<T>, dim3((p.width + LC - 1) / LC, num_seqs), dim3(LW * 32), (size_t)0, stream, p));
  PG_LAUNCH_CHECK();
  return PG_OK;
}

}  // namespace

// gates f32 [tokens, blocks, 2 part] contiguous, part = width / blocks; gate_bias f32 of one row; u, y, out: rows [width] of the activation type
// with their own strides; lam, y_bias f32 [width]; state f32 [slots, width].
extern "C" int pg_gated_lru(const void* gates, const void* gate_bias, const void* u, long long ldu, const void* lam, const void* y, long long ldy, const void* y_bias, void* state, void* out, long long ldo,
                            const void* q_indptr, const void* slots, int num_seqs, int width, int blocks, float scale, int max_q_len, int is_f32, cudaStream_t stream) {
  PG_REQUIRE(blocks >= 1 && width >= 1 && width % blocks == 0, "gated_lru: %d channels in %d blocks", width, blocks);
  PG_REQUIRE(num_seqs <= 65535 && width < (1 << 27) && ldu < (1ll << 28) && ldy < (1ll << 28) && ldo < (1ll << 28), "gated_lru: %d sequences, rows of %lld / %lld / %lld", num_seqs, ldu, ldy, ldo);
  if (num_seqs == 0) return PG_OK;
#define PG_LRU(T)                                                                                                                                                                         \
  run_lru<T>(LruArgs<T>{(const float*)gates, (const float*)gate_bias, (const T*)u, ldu, (const float*)lam, (const T*)y, ldy, (const float*)y_bias, (float*)state, (T*)out, ldo, \
                        (const int*)q_indptr, (const int*)slots, width, width / blocks, scale},                                                                                     \
             num_seqs, max_q_len, stream)
  return is_f32 ? PG_LRU(float) : PG_LRU(bf16);
#undef PG_LRU
}
