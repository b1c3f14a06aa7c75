// Attention pieces for layers whose head sizes, norms and masks are runtime parameters (bf16 and f32).
//
//  * row_norm_rope_append: RMS norm over the whole query (and key) projection row of a token, rotation of neighbouring
//    pairs (2i, 2i + 1) of the first `rot` entries of every head with f32 cos / sin tables, then the queries go to a
//    dense buffer and keys and values to the token's slot of the paged cache.  One CTA per token.  Without keys (a layer
//    that reads another layer's cache) only the queries are made.
//  * head_norm_append: RMS norm of every query and key head with a weight shared by the heads (or one per query head), queries
//    times a factor per position; queries go to a dense buffer, keys and values (untouched; they may be the key projection
//    itself) to the cache.  The projections' biases, if there are any, are added first.
//  * attention_plain: one CTA per (query row, head) on the CUDA cores, keys in chunks of 128 with an online softmax; any
//    head size, value size and group.  It is the 32-bit path, and the path of head sizes the tensor-core kernels
//    (attention.cu, attention_tc.cu) do not address.
//
// Score = dot(q, k) * scale, then softcap * tanh(score / softcap) when a cap is given, less slope[head] * distance when
// slopes are given, over the last `window` keys (0: all); the head's output is multiplied by out_scale and by
// sigmoid(gate[token, head]) when a gate is given.  Cache page of one layer: [page_size, kv_heads, dim] keys, then
// [page_size, kv_heads, vdim] values.
#include "api.h"
#include "common.cuh"
#include "types.cuh"

namespace {

template <typename T, int V>
__global__ void __launch_bounds__(256) row_norm_rope_append_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long long ld, const float* __restrict__ q_w,
                                                                   const float* __restrict__ k_w, const float* __restrict__ cos, const float* __restrict__ sin, int rot, int max_pos,
                                                                   const int* __restrict__ positions, const int* __restrict__ slots, T* __restrict__ q_out, T* __restrict__ kv, int hq, int hkv,
                                                                   int dim, int vdim, int page_size, long long num_pages, float eps, uint32_t* status) {
  PG_PDL_ENTRY();
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const int tid = threadIdx.x;
  const T* qr = q + t * ld;
  const T* kr = k ? k + t * ld : nullptr;
  const int nq = hq * dim / V, nk = k ? hkv * dim / V : 0;
  constexpr int KEEP = 4;
  float qv[KEEP][V], kv1[V];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int c = 0; c < KEEP; ++c) {
    const int i = tid + c * 256;
    if (i < nq) {
      load_vec<V>(qr + i * V, qv[c]);
#pragma unroll
      for (int j = 0; j < V; ++j) sq += qv[c][j] * qv[c][j];
    }
  }
  for (int i = tid + KEEP * 256; i < nq; i += 256) {
    float f[V];
    load_vec<V>(qr + i * V, f);
#pragma unroll
    for (int j = 0; j < V; ++j) sq += f[j] * f[j];
  }
  for (int i = tid; i < nk; i += 256) {
    float f[V];
    load_vec<V>(kr + i * V, f);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      if (i == tid) kv1[j] = f[j];
      sk += f[j] * f[j];
    }
  }
  int pos = positions[t];
  if (pos < 0 || pos >= max_pos) {
    if (tid == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (51u << 8));
    pos = pos < 0 ? 0 : max_pos - 1;
  }
  const long long slot = slots[t];
  const bool slot_ok = slot >= 0 && slot < num_pages * page_size;
  if (k && !slot_ok && tid == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (52u << 8));
  sq = block_sum(sq, red);
  if (k) sk = block_sum(sk, red);
  const float iq = rsqrtf(sq / (float)(hq * dim) + eps), ik = k ? rsqrtf(sk / (float)(hkv * dim) + eps) : 0.f;
  const float* cs = cos + (long long)pos * (rot / 2);
  const float* sn = sin + (long long)pos * (rot / 2);
  // elements e .. e + V - 1 of a projection row, normalised and rotated
  auto finish = [&](float* f, const T* row, const float* w, float inv, int e) {
    const int d = e % dim;
    if constexpr (V > 1) {  // dim is a multiple of V, so pairs and heads do not straddle the vector
      float wf[V];
      load_vec<V>(w + e, wf);
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] *= inv * wf[j];
#pragma unroll
      for (int j = 0; j < V; j += 2) {
        if (d + j < rot) {
          const float c = cs[(d + j) >> 1], s = sn[(d + j) >> 1];
          const float a = f[j] * c - f[j + 1] * s, b = f[j + 1] * c + f[j] * s;
          f[j] = a, f[j + 1] = b;
        }
      }
    } else {
      float a = f[0] * inv * w[e];
      if (d < rot) {
        const int pe = (d & 1) ? e - 1 : e + 1;
        const float b = to_f32(row[pe]) * inv * w[pe], c = cs[d >> 1], s = sn[d >> 1];
        a = (d & 1) ? a * c + b * s : a * c - b * s;
      }
      f[0] = a;
    }
  };
  T* qo = q_out + t * hq * dim;
#pragma unroll
  for (int c = 0; c < KEEP; ++c) {
    const int i = tid + c * 256;
    if (i < nq) {
      finish(qv[c], qr, q_w, iq, i * V);
      store_vec<V>(qo + i * V, qv[c]);
    }
  }
  for (int i = tid + KEEP * 256; i < nq; i += 256) {
    float f[V];
    load_vec<V>(qr + i * V, f);
    finish(f, qr, q_w, iq, i * V);
    store_vec<V>(qo + i * V, f);
  }
  if (!k || !slot_ok) return;
  const long long page = slot / page_size, off = slot % page_size;
  T* kpage = kv + page * page_size * hkv * (dim + vdim);
  T* kd = kpage + off * hkv * dim;
  T* vd = kpage + (long long)page_size * hkv * dim + off * hkv * vdim;
  for (int i = tid; i < nk; i += 256) {
    float f[V];
    if (i == tid) {
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] = kv1[j];
    } else {
      load_vec<V>(kr + i * V, f);
    }
    finish(f, kr, k_w, ik, i * V);
    store_vec<V>(kd + i * V, f);
  }
  const T* vr = v + t * ld;
  for (int i = tid; i < hkv * vdim / V; i += 256) {
    float f[V];
    load_vec<V>(vr + i * V, f);
    store_vec<V>(vd + i * V, f);
  }
}

// TPR threads (16 or 32) per unit of a token: hq query heads, hkv key heads, hkv value heads.
template <typename T, int V, int TPR>
__global__ void __launch_bounds__(256) head_norm_append_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long long ld, const float* __restrict__ q_w, int q_w_heads,
                                                               const float* __restrict__ k_w, const float* __restrict__ q_b, const float* __restrict__ k_b, const float* __restrict__ v_b, const float* __restrict__ temp, int max_pos, const int* __restrict__ positions, const int* __restrict__ slots, T* __restrict__ q_out,
                                                               T* __restrict__ kv, int hq, int hkv, int dim, int vdim, int page_size, long long num_pages, float eps, uint32_t* status) {
  PG_PDL_ENTRY();
  const long long t = blockIdx.x;
  const int me = threadIdx.x % TPR, units = hq + 2 * hkv;
  float factor = 1.f;
  if (temp) {
    int pos = positions[t];
    if (pos < 0 || pos >= max_pos) {
      if (threadIdx.x == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (57u << 8));
      pos = pos < 0 ? 0 : max_pos - 1;
    }
    factor = temp[pos];
  }
  const long long slot = slots[t];
  const bool slot_ok = slot >= 0 && slot < num_pages * page_size;
  if (!slot_ok && threadIdx.x == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (58u << 8));
  const long long page = slot / page_size, off = slot % page_size;
  T* kpage = kv + page * page_size * hkv * (dim + vdim);
  for (int u0 = 0; u0 < units; u0 += 256 / TPR) {  // all lanes of a warp take part in the sums
    const int u = u0 + threadIdx.x / TPR;
    const bool live = u < units && (u < hq || slot_ok), value = u >= hq + hkv;
    const int h = u < hq ? u : value ? u - hq - hkv : u - hq, n = live ? (value ? vdim : dim) / V : 0;
    const T* src = u < hq ? q + t * ld + (long long)h * dim : value ? v + t * ld + (long long)h * vdim : k + t * ld + (long long)h * dim;
    T* dst = u < hq ? q_out + (t * hq + h) * dim : value ? kpage + (long long)page_size * hkv * dim + (off * hkv + h) * vdim : kpage + (off * hkv + h) * dim;
    const float* bias = u < hq ? q_b : value ? v_b : k_b;
    if (bias) bias += h * (value ? vdim : dim);
    float f[V], ss = 0.f;
    auto get = [&](int i) {
      load_vec<V>(src + i * V, f);
      if (bias) {
        float bf[V];
        load_vec<V>(bias + i * V, bf);
#pragma unroll
        for (int j = 0; j < V; ++j) f[j] += bf[j];
      }
    };
    for (int i = me; i < n; i += TPR) {
      get(i);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += f[j] * f[j];
    }
#pragma unroll
    for (int o = TPR / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = rsqrtf(ss / (float)dim + eps) * (u < hq ? factor : 1.f);
    const float* w = u < hq ? q_w + (q_w_heads ? h * dim : 0) : k_w;
    for (int i = me; i < n; i += TPR) {
      if (n > TPR) get(i);
      if (!value) {
        float wf[V];
        load_vec<V>(w + i * V, wf);
#pragma unroll
        for (int j = 0; j < V; ++j) f[j] *= inv * wf[j];
      }
      store_vec<V>(dst + i * V, f);
    }
  }
}

constexpr int PL_KEYS = 128;  // keys per chunk, one per thread
constexpr int PL_VMAX = 8;    // value columns per thread: vdim <= 1024

template <typename T>
__global__ void __launch_bounds__(128) attention_plain_kernel(const T* __restrict__ q, const T* __restrict__ kv, T* __restrict__ out, const int* __restrict__ q_indptr, const int* __restrict__ kv_lens,
                                                              const int* __restrict__ table, int table_stride, int num_seqs, int hq, int hkv, int dim, int vdim, int page_size, long long num_pages,
                                                              float scale, float softcap, const T* __restrict__ gate, long long ld_gate, int window, const float* __restrict__ slopes, float out_scale,
                                                              long long ld_out) {
  PG_PDL_ENTRY();
  extern __shared__ float sm[];
  float* sq = sm;         // [dim]
  float* sp = sm + dim;   // [PL_KEYS]
  __shared__ float red[4];
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = h / (hq / hkv);
  // the row's sequence: the last one that starts at or before it
  int lo = 0, hi = num_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (q_indptr[mid] <= t) lo = mid;
    else hi = mid - 1;
  }
  const int b = lo;
  const int n = kv_lens[b] - (q_indptr[b + 1] - 1 - t);  // visible keys: positions 0 .. the row's own
  const int* pages = table + (long long)b * table_stride;
  for (int i = tid; i < dim; i += 128) sq[i] = to_f32(q[((long long)t * hq + h) * dim + i]);
  __syncthreads();
  const long long page_elems = (long long)page_size * hkv * (dim + vdim), v_plane = (long long)page_size * hkv * dim;
  float m = -INFINITY, l = 0.f, acc[PL_VMAX];
#pragma unroll
  for (int i = 0; i < PL_VMAX; ++i) acc[i] = 0.f;
  const int first = window > 0 ? max(0, n - window) : 0;  // visible keys: first .. n - 1
  const float slope = slopes ? slopes[h] : 0.f;
  for (int k0 = first; k0 < n; k0 += PL_KEYS) {
    const int key = k0 + tid;
    float s = -INFINITY;
    if (key < n) {
      const T* kr = kv + pages[key / page_size] * page_elems + ((long long)(key % page_size) * hkv + g) * dim;
      float a = 0.f;
      for (int i = 0; i < dim; ++i) a = fmaf(sq[i], to_f32(kr[i]), a);
      s = a * scale;
      if (softcap > 0.f) s = softcap * tanh_full(s / softcap);
      s -= slope * (float)(n - 1 - key);
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
      const T* vr = kv + pages[kk / page_size] * page_elems + v_plane + ((long long)(kk % page_size) * hkv + g) * vdim;
      const float pj = sp[j];
#pragma unroll
      for (int i = 0; i < PL_VMAX; ++i)
        if (tid + 128 * i < vdim) acc[i] = fmaf(pj, to_f32(vr[tid + 128 * i]), acc[i]);
    }
    __syncthreads();
  }
  float f = l > 0.f ? out_scale / l : 0.f;
  if (gate) f /= 1.f + __expf(-to_f32(gate[(long long)t * ld_gate + h]));
#pragma unroll
  for (int i = 0; i < PL_VMAX; ++i)
    if (tid + 128 * i < vdim) out[t * ld_out + (long long)h * vdim + tid + 128 * i] = from_f32<T>(acc[i] * f);
}

}  // namespace

extern "C" int pg_row_norm_rope_append(const void* q, const void* k, const void* v, long long ld, const void* q_w, const void* k_w, const void* cos, const void* sin, int rot, int max_pos,
                                       const void* positions, const void* slots, void* q_out, void* kv, int tokens, int hq, int hkv, int dim, int vdim, int page_size, long long num_pages, float eps,
                                       int is_f32, void* status, cudaStream_t stream) {
  PG_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= dim, "row_norm_rope: %d rotated entries of a head of %d", rot, dim);
  PG_REQUIRE((k == nullptr) == (v == nullptr) && (k == nullptr || (kv && k_w)), "row_norm_rope: keys, values, their norm weight and the cache come together");
  if (tokens == 0) return PG_OK;
  const bool v8 = dim % 8 == 0 && vdim % 8 == 0 && ld % 8 == 0 && ((((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)q_out | (uintptr_t)kv | (uintptr_t)q_w | (uintptr_t)k_w) & 15) == 0);
#define PG_RNR(T, V)                                                                                                                                                                                  \
  launch_pdl(row_norm_rope_append_kernel<T, V>, dim3(tokens), dim3(256), (size_t)0, stream, (const T*)q, (const T*)k, (const T*)v, ld, (const float*)q_w, (const float*)k_w, (const float*)cos,        \
             (const float*)sin, rot, max_pos, (const int*)positions, (const int*)slots, (T*)q_out, (T*)kv, hq, hkv, dim, vdim, page_size, num_pages, eps, (uint32_t*)status)
  if (is_f32)
    PG_CUDA(PG_RNR(float, 1));
  else
    PG_CUDA(v8 ? PG_RNR(bf16, 8) : PG_RNR(bf16, 1));
#undef PG_RNR
  PG_LAUNCH_CHECK();
  return PG_OK;
}

// q, k, v: columns of rows of stride ld; q_w f32 [dim], or [hq, dim] with q_w_heads; q_b, k_b, v_b: biases in f32 (or null); temp f32
// [max_pos] (or null); cache as above.
extern "C" int pg_head_norm_append(const void* q, const void* k, const void* v, long long ld, const void* q_w, int q_w_heads, const void* k_w, const void* q_b, const void* k_b, const void* v_b, const void* temp, int max_pos, const void* positions, const void* slots,
                                   void* q_out, void* kv, int tokens, int hq, int hkv, int dim, int vdim, int page_size, long long num_pages, float eps, int is_f32, void* status, cudaStream_t stream) {
  PG_REQUIRE(hq >= 1 && hkv >= 1 && dim >= 1 && vdim >= 1 && (temp == nullptr || max_pos > 0), "head_norm_append: heads %d / %d of %d / %d columns", hq, hkv, dim, vdim);
  if (tokens == 0) return PG_OK;
  const uintptr_t all = (uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)q_out | (uintptr_t)kv | (uintptr_t)q_w | (uintptr_t)k_w | (uintptr_t)q_b | (uintptr_t)k_b | (uintptr_t)v_b;
  const bool v8 = dim % 8 == 0 && vdim % 8 == 0 && ld % 8 == 0 && (all & 15) == 0;
#define PG_HN(T, V, TPR)                                                                                                                                                                            \
  launch_pdl(head_norm_append_kernel<T, V, TPR>, dim3(tokens), dim3(256), (size_t)0, stream, (const T*)q, (const T*)k, (const T*)v, ld, (const float*)q_w, q_w_heads, (const float*)k_w, (const float*)q_b, (const float*)k_b, (const float*)v_b, (const float*)temp, max_pos, \
             (const int*)positions, (const int*)slots, (T*)q_out, (T*)kv, hq, hkv, dim, vdim, page_size, num_pages, eps, (uint32_t*)status)
  if (is_f32)
    PG_CUDA(PG_HN(float, 1, 32));
  else
    PG_CUDA(v8 ? (dim <= 128 && vdim <= 128 ? PG_HN(bf16, 8, 16) : PG_HN(bf16, 8, 32)) : PG_HN(bf16, 1, 32));
#undef PG_HN
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_attention_plain(const void* q, const void* kv, void* out, const void* q_indptr, const void* kv_lens, const void* table, int table_stride, int tokens, int num_seqs, int hq, int hkv,
                                  int dim, int vdim, int page_size, long long num_pages, float scale, float softcap, const void* gate, long long ld_gate, int window, const void* slopes, float out_scale, long long ld_out,
                                  int is_f32, cudaStream_t stream) {
  PG_REQUIRE(hq % hkv == 0 && dim <= 8192 && vdim <= 128 * PL_VMAX, "attention_plain: heads %d / %d, sizes %d / %d not supported", hq, hkv, dim, vdim);
  if (tokens == 0) return PG_OK;
  const size_t smem = (size_t)(dim + PL_KEYS) * 4;
#define PG_AP(T)                                                                                                                                                                                    \
  launch_pdl(attention_plain_kernel<T>, dim3(tokens, hq), dim3(128), smem, stream, (const T*)q, (const T*)kv, (T*)out, (const int*)q_indptr, (const int*)kv_lens, (const int*)table, table_stride,    \
             num_seqs, hq, hkv, dim, vdim, page_size, num_pages, scale, softcap, (const T*)gate, ld_gate, window, (const float*)slopes, out_scale, ld_out)
  if (is_f32)
    PG_CUDA(PG_AP(float));
  else
    PG_CUDA(PG_AP(bf16));
#undef PG_AP
  PG_LAUNCH_CHECK();
  return PG_OK;
}
