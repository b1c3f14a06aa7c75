// Linear attention with a decay per token and key channel (WKV): the token shift in front of its projections.
//
//  * token_mix: every projection of the layer reads its own mix of a token's row with the previous one's,
//      out[t, i] = h[t] + (h[t - 1] - h[t]) * mu[i].
//    The row in front of a step's first row comes from the request's slot, which then takes the step's last row.  A thread
//    owns V columns for a run of rows, so the mix weights stay in registers and each row is read once.
#include "api.h"
#include "common.cuh"
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

}  // namespace

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
