// Row kernels around a residual stream that is kept in 32 bits, for bf16 and f32 activations.
//
//  * embed_rows: table row -> f32 stream row (+ a copy in the activation type for the next projection).
//  * embed_pairs_norm: scaled table row plus the row of the pair (previous token, token) -> f32 stream row and its RMS norm.
//    The previous token of a step's first row comes from the request's slot, which then takes the step's last token.
//  * residual_norm: the norm before the sublayer.  x += mult * y on the f32 stream, and the RMS norm of the sum, which the
//    next sublayer reads, in the same pass.  y is a projection's output, or the weighted sum of a token's expert rows plus a
//    further row times the sigmoid of a number per token (an expert that every token takes).
//  * post_norm: the norm after the sum.  s = alpha * x + y; x = s / sqrt(mean(s^2) + eps) * w.  The stream x is read and
//    written in f32, y is a projection's output (f32 or bf16), and the activation-type copy that the next projection
//    reads is written in the same pass.  Without y and with alpha = 1 it is a plain RMS norm of the stream.
//  * add_layer_norm: the norm of a sublayer's output before the sum.  x += (y - mean(y)) / sqrt(mean((y - mean)^2) + eps) * w
//    on the f32 stream, with the activation-type copy of the new stream written in the same pass.  y is a projection's
//    output, or the weighted sum of a token's expert rows, which is then formed here instead of by a kernel of its own.
//    With y = x and no sum it is the plain layer norm of the stream.
//  * gated_row_norm: RMS norm over a row (one head, or all heads of a token at once), times a weight, times the sigmoid or
//    the SiLU of a gate row that may lie inside a wider projection output; or the gate in front of the norm.
//  * glu_rows: silu(gate) * up or gelu(gate) * up on f32 rows; softcap_f32: cap * tanh(x / cap) on f32 values; tanh_rows; xielu_rows.
//  * gemm_simt: y = x w^T on the CUDA cores with f32 accumulation, for f32 operands (the 32-bit mode) and for bf16
//    problems whose rows the TMA kernels cannot address (an inner size that is not a multiple of 8).  head_gemm_simt is the
//    same per attention head (strided operands, sigmoid gate on the output), expert_gemm_simt per expert over sorted rows.
//  * short_conv: causal depthwise convolution of any length over ragged sequences with carried inputs; biases on the inputs and on
//    the sum and a SiLU are optional.
#include "api.h"
#include "common.cuh"
#include "types.cuh"

namespace {

template <typename TI, typename TO>
__global__ void __launch_bounds__(256) embed_rows_kernel(const TI* __restrict__ table, long long ldt, const int* __restrict__ ids, float* __restrict__ x, TO* __restrict__ xt, long long ldxt,
                                                         int width, long long rows, uint32_t* status) {
  PG_PDL_ENTRY();
  const int t = blockIdx.x;
  long long id = ids[t];
  if (id < 0 || id >= rows) {
    if (threadIdx.x == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (50u << 8));
    id = 0;
  }
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float v = to_f32(table[id * ldt + i]);
    if (x) x[(long long)t * width + i] = v;
    if (xt) xt[(long long)t * ldxt + i] = from_f32<TO>(v);
  }
}

// One CTA per row.  `unit_seq[t]`: sequence of row t.  The CTA of a sequence's first row is the only one that touches its slot.
template <typename T, typename TO, int V>
__global__ void __launch_bounds__(256) embed_pairs_norm_kernel(const T* __restrict__ table, long long ldt, const T* __restrict__ pairs, long long ldp, const int* __restrict__ ids, const int* __restrict__ unit_seq,
                                                               const int* __restrict__ q_indptr, const int* __restrict__ slots, int* __restrict__ carried, float scale, long long buckets, long long mul_prev,
                                                               long long mul_cur, const float* __restrict__ w, float* __restrict__ x, TO* __restrict__ xt, int width, long long rows, float eps,
                                                               uint32_t* status) {
  PG_PDL_ENTRY();
  __shared__ float red[32];
  __shared__ long long s_pair;
  const int t = blockIdx.x;
  long long id = ids[t];
  if (threadIdx.x == 0) {
    if (id < 0 || id >= rows) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (56u << 8));
    if (pairs) {
      const int b = unit_seq[t], q0 = q_indptr[b], slot = slots[b];
      long long prev = t > q0 ? (long long)ids[t - 1] : slot >= 0 ? (long long)carried[slot] - 1 : -1;
      if (t == q0 && slot >= 0) carried[slot] = ids[q_indptr[b + 1] - 1] + 1;
      const long long sum = prev * mul_prev + (id < 0 ? 0 : id) * mul_cur;
      s_pair = prev < 0 || sum < 0 ? buckets : sum % buckets;
    }
  }
  if (id < 0 || id >= rows) id = 0;
  __syncthreads();
  const T* row = table + id * ldt;
  const T* pair = pairs ? pairs + s_pair * ldp : nullptr;
  constexpr int KEEP = 8;
  const int nv = width / V;
  float s[KEEP][V], ss = 0.f;
  auto sum_at = [&](int i, float* o) {
    load_vec<V>(row + i * V, o);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] *= scale;
    if (pair) {
      float f[V];
      load_vec<V>(pair + i * V, f);
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] += f[j];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) ss += o[j] * o[j];
    store_vec<V>(x + (long long)t * width + i * V, o);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k)
    if (threadIdx.x + k * 256 < nv) sum_at(threadIdx.x + k * 256, s[k]);
  for (int i = threadIdx.x + KEEP * 256; i < nv; i += 256) {  // wider rows: read back below
    float o[V];
    sum_at(i, o);
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)width + eps);
  auto put = [&](int i, const float* o) {
    float wf[V], r[V];
    load_vec<V>(w + i * V, wf);
#pragma unroll
    for (int j = 0; j < V; ++j) r[j] = o[j] * inv * wf[j];
    store_vec<V>(xt + (long long)t * width + i * V, r);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k)
    if (threadIdx.x + k * 256 < nv) put(threadIdx.x + k * 256, s[k]);
  for (int i = threadIdx.x + KEEP * 256; i < nv; i += 256) {
    float o[V];
    load_vec<V>(x + (long long)t * width + i * V, o);
    put(i, o);
  }
}

// One CTA per row; V consecutive elements per access (4 when every row allows it, else 1).
template <typename TY, typename TO, int V>
__global__ void __launch_bounds__(256) post_norm_kernel(const TY* __restrict__ y, long long ldy, const float* __restrict__ xin, float* __restrict__ x, float alpha, const float* __restrict__ w, TO* __restrict__ xt,
                                                        long long ldxt, int width, float eps) {
  PG_PDL_ENTRY();
  __shared__ float red[32];
  constexpr int KEEP = 8;
  const long long row = blockIdx.x;
  const int nv = width / V;
  const float* xi = xin + row * width;
  const TY* yr = y ? y + row * ldy : nullptr;
  float s[KEEP][V];
  float ss = 0.f;
  auto sum_at = [&](int i, float* o) {
    load_vec<V>(xi + i * V, o);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] *= alpha;
    if (yr) {
      float f[V];
      load_vec<V>(yr + i * V, f);
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] += f[j];
    }
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < nv) {
      sum_at(i, s[k]);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += s[k][j] * s[k][j];
    }
  }
  for (int i = threadIdx.x + KEEP * 256; i < nv; i += 256) {  // wider rows: summed again below
    float o[V];
    sum_at(i, o);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += o[j] * o[j];
  }
  ss = block_sum(ss, red);
  const float inv = rsqrtf(ss / (float)width + eps);
  auto put = [&](int i, float* o) {
    float wf[V];
    load_vec<V>(w + i * V, wf);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = o[j] * inv * wf[j];
    if (x) store_vec<V>(x + row * width + i * V, o);
    if (xt) store_vec<V>(xt + row * ldxt + i * V, o);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < nv) put(i, s[k]);
  }
  for (int i = threadIdx.x + KEEP * 256; i < nv; i += 256) {
    float o[V];
    sum_at(i, o);
    put(i, o);
  }
}

// A row's y: a row of one matrix, or sum_j weights[j] * rows[pos[j]] over the token's k expert rows (rows of one matrix
// sorted by expert; pos < 0: none).
template <typename TY>
struct RowSource {
  const TY* y;
  long long ld;
  const int* pos;
  const float* weights;
  int k;
  template <int V>
  __device__ __forceinline__ void load(long long row, int at, float* o) const {
    if (pos == nullptr) {
      load_vec<V>(y + row * ld + at, o);
      return;
    }
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = 0.f;
    for (int s = 0; s < k; ++s) {
      const int r = pos[row * k + s];
      if (r < 0) continue;
      const float w = weights[row * k + s];
      float f[V];
      load_vec<V>(y + r * ld + at, f);
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] = fmaf(w, f[j], o[j]);
    }
  }
};

// One CTA per row.  x += mult * (src row + sigmoid(extra_gate[row]) * extra row); xt = rms_norm(x) * w.
template <typename TY, typename TO, int V>
__global__ void __launch_bounds__(256) residual_norm_kernel(const RowSource<TY> src, const void* __restrict__ extra, int extra_f32, long long lde, const float* __restrict__ extra_gate, long long ldg,
                                                            float* __restrict__ x, float mult, const float* __restrict__ w, TO* __restrict__ xt, long long ldxt, int width, float eps) {
  PG_PDL_ENTRY();
  __shared__ float red[32];
  constexpr int KEEP = 8;
  const long long row = blockIdx.x;
  const int nv = width / V;
  float* xr = x + row * width;
  const float gate = extra ? (extra_gate ? 1.f / (1.f + __expf(-extra_gate[row * ldg])) : 1.f) : 0.f;
  float s[KEEP][V], ss = 0.f;
  auto sum_at = [&](int i, float* o) {
    float y[V];
    src.template load<V>(row, i * V, y);
    if (extra) {
      float f[V];
      if (extra_f32)
        load_vec<V>(reinterpret_cast<const float*>(extra) + row * lde + i * V, f);
      else
        load_vec<V>(reinterpret_cast<const bf16*>(extra) + row * lde + i * V, f);
#pragma unroll
      for (int j = 0; j < V; ++j) y[j] = fmaf(gate, f[j], y[j]);
    }
    load_vec<V>(xr + i * V, o);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      o[j] = fmaf(mult, y[j], o[j]);
      ss += o[j] * o[j];
    }
    store_vec<V>(xr + i * V, o);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k)
    if (threadIdx.x + k * 256 < nv) sum_at(threadIdx.x + k * 256, s[k]);
  for (int i = threadIdx.x + KEEP * 256; i < nv; i += 256) {  // wider rows: read back below
    float o[V];
    sum_at(i, o);
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)width + eps);
  auto put = [&](int i, const float* o) {
    float wf[V], r[V];
    load_vec<V>(w + i * V, wf);
#pragma unroll
    for (int j = 0; j < V; ++j) r[j] = o[j] * inv * wf[j];
    store_vec<V>(xt + row * ldxt + i * V, r);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k)
    if (threadIdx.x + k * 256 < nv) put(threadIdx.x + k * 256, s[k]);
  for (int i = threadIdx.x + KEEP * 256; i < nv; i += 256) {
    float o[V];
    load_vec<V>(xr + i * V, o);
    put(i, o);
  }
}

// One CTA per row.  x (f32 stream) is read and written; x == nullptr: only the norm goes to xt.
template <typename TY, typename TO, int V>
__global__ void __launch_bounds__(256) add_layer_norm_kernel(const RowSource<TY> src, float* __restrict__ x, const float* __restrict__ w, TO* __restrict__ xt, long long ldxt, int width, float eps) {
  PG_PDL_ENTRY();
  __shared__ float red[32];
  constexpr int KEEP = 8;
  const long long row = blockIdx.x;
  const int nv = width / V;
  float v[KEEP][V], sum = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < nv) {
      src.template load<V>(row, i * V, v[k]);
#pragma unroll
      for (int j = 0; j < V; ++j) sum += v[k][j];
    }
  }
  for (int i = threadIdx.x + KEEP * 256; i < nv; i += 256) {  // wider rows: read again below
    float o[V];
    src.template load<V>(row, i * V, o);
#pragma unroll
    for (int j = 0; j < V; ++j) sum += o[j];
  }
  const float mean = block_sum(sum, red) / (float)width;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k)
    if (threadIdx.x + k * 256 < nv) {
#pragma unroll
      for (int j = 0; j < V; ++j) ss += (v[k][j] - mean) * (v[k][j] - mean);
    }
  for (int i = threadIdx.x + KEEP * 256; i < nv; i += 256) {
    float o[V];
    src.template load<V>(row, i * V, o);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += (o[j] - mean) * (o[j] - mean);
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)width + eps);
  auto put = [&](int i, float* o) {
    float wf[V];
    load_vec<V>(w + i * V, wf);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = (o[j] - mean) * inv * wf[j];
    if (x) {
      float xf[V];
      load_vec<V>(x + row * width + i * V, xf);
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] += xf[j];
      store_vec<V>(x + row * width + i * V, o);
    }
    if (xt) store_vec<V>(xt + row * ldxt + i * V, o);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < nv) put(i, v[k]);
  }
  for (int i = threadIdx.x + KEEP * 256; i < nv; i += 256) {
    float o[V];
    src.template load<V>(row, i * V, o);
    put(i, o);
  }
}

// TPR threads per row (16, 32 or 256); row r = token * heads + head; the gate row of (token, head) is gate + token * ldg + head * dim.
template <typename T, int V, int TPR>
__global__ void __launch_bounds__(256) gated_row_norm_kernel(const T* __restrict__ x, const T* __restrict__ gate, long long ldg, const float* __restrict__ w, T* __restrict__ y, long long rows, int heads, int dim,
                                                             float eps, int silu, int w_heads, int gate_first) {
  PG_PDL_ENTRY();
  __shared__ float red[32];
  const long long row = TPR == 256 ? (long long)blockIdx.x : (long long)blockIdx.x * (256 / TPR) + threadIdx.x / TPR;
  const int me = threadIdx.x % TPR;
  const bool live = row < rows;  // with TPR == 256 the grid has no spare blocks
  const T* xr = x + row * dim;
  const T* gr = gate + (row / heads) * ldg + (row % heads) * dim;
  if (w_heads) w += (row % heads) * dim;  // a weight per head
  constexpr int KEEP = 4;
  const int nv = live ? dim / V : 0;
  float f[KEEP][V], ss = 0.f;
  auto get = [&](int i, float* o) {
    load_vec<V>(xr + i * V, o);
    if (gate_first) {
      float g[V];
      load_vec<V>(gr + i * V, g);
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] *= (silu ? g[j] : 1.f) / (1.f + __expf(-g[j]));
    }
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = me + k * TPR;
    if (i < nv) {
      get(i, f[k]);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += f[k][j] * f[k][j];
    }
  }
  for (int i = me + KEEP * TPR; i < nv; i += TPR) {
    float o[V];
    get(i, o);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += o[j] * o[j];
  }
  if (TPR == 256) {
    ss = block_sum(ss, red);
  } else {
#pragma unroll
    for (int o = TPR / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  }
  const float inv = rsqrtf(ss / (float)dim + eps);
  auto put = [&](int i, const float* o) {
    float g[V], wf[V], r[V];
    load_vec<V>(w + i * V, wf);
    if (gate_first) {
#pragma unroll
      for (int j = 0; j < V; ++j) r[j] = o[j] * inv * wf[j];
    } else {
      load_vec<V>(gr + i * V, g);
#pragma unroll
      for (int j = 0; j < V; ++j) r[j] = o[j] * inv * wf[j] * (silu ? g[j] : 1.f) / (1.f + __expf(-g[j]));
    }
    store_vec<V>(y + row * dim + i * V, r);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = me + k * TPR;
    if (i < nv) put(i, f[k]);
  }
  for (int i = me + KEEP * TPR; i < nv; i += TPR) {
    float o[V];
    get(i, o);
    put(i, o);
  }
}

template <typename TO>
__global__ void xielu_rows_kernel(const float* __restrict__ x, TO* __restrict__ y, const float* __restrict__ act, long long n) {
  PG_PDL_ENTRY();
  const float a = act[0], b = act[1];
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) y[i] = from_f32<TO>(xielu(x[i], a, b));
}

__global__ void glu_rows_kernel(const float* __restrict__ gu, float* __restrict__ out, int rows, int inter, long long ldin, int gelu) {
  PG_PDL_ENTRY();
  const long long total = (long long)rows * inter;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / inter, c = i % inter;
    const float g = gu[r * ldin + c], u = gu[r * ldin + inter + c];
    out[i] = glu_act(g, gelu) * u;
  }
}

template <typename T>
__global__ void tanh_rows_kernel(const T* __restrict__ x, T* __restrict__ y, long long n) {
  PG_PDL_ENTRY();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) y[i] = from_f32<T>(tanh_full(to_f32(x[i])));
}

__global__ void softcap_f32_kernel(const float* __restrict__ x, float* __restrict__ y, long long n, float cap) {
  PG_PDL_ENTRY();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) y[i] = cap * tanh_full(x[i] / cap);
}

// 64 x 64 output tile, 256 threads of 4 x 4 outputs, 16-deep k steps: acc = x rows [t0, T) times w rows [m0, M).
// `xrow(t)` is the row of x that output row t reads.
template <typename TX, typename XRow>
__device__ __forceinline__ void simt_tile(const TX* __restrict__ x, const TX* __restrict__ w, int t0, int T, int m0, int M, int K, long long ldx, long long ldw, XRow xrow, float (&acc)[4][4]) {
  __shared__ float xs[16][68], ws[16][68];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int r = i >> 4, k = i & 15;
      const bool kin = k0 + k < K;
      xs[k][r] = (kin && t0 + r < T) ? to_f32(x[(long long)xrow(t0 + r) * ldx + k0 + k]) : 0.f;
      ws[k][r] = (kin && m0 + r < M) ? to_f32(w[(long long)(m0 + r) * ldw + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]), b = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
}

template <typename TX, typename TY>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const TX* __restrict__ x, const TX* __restrict__ w, TY* __restrict__ y, int T, int M, int K, long long ldx, long long ldw, long long ldy) {
  PG_PDL_ENTRY();
  const int m0 = blockIdx.x * 64, t0 = blockIdx.y * 64;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  simt_tile(x, w, t0, T, m0, M, K, ldx, ldw, [](int t) { return t; }, acc);
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, m = m0 + tx * 4 + j;
      if (t < T && m < M) y[(long long)t * ldy + m] = from_f32<TY>(acc[i][j]);
    }
}

// Head h (grid z): y[t, h, :] = x[t, h, :] w[h]^T, times sigmoid(gate[t, h, :]) when a gate is given.
template <typename T, typename TY>
__global__ void __launch_bounds__(256) head_gemm_simt_kernel(const T* __restrict__ x, long long ldx, long long x_head, const T* __restrict__ w, TY* __restrict__ y, long long ldy, long long y_head,
                                                             const T* __restrict__ gate, long long ldg, long long g_head, int rows, int M, int K) {
  PG_PDL_ENTRY();
  const int m0 = blockIdx.x * 64, t0 = blockIdx.y * 64, h = blockIdx.z;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  simt_tile(x + h * x_head, w + (long long)h * M * K, t0, rows, m0, M, K, ldx, (long long)K, [](int t) { return t; }, acc);
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, m = m0 + tx * 4 + j;
      if (t >= rows || m >= M) continue;
      float v = acc[i][j];
      if (gate) v /= 1.f + __expf(-to_f32(gate[(long long)t * ldg + h * g_head + m]));
      y[(long long)t * ldy + h * y_head + m] = from_f32<TY>(v);
    }
}

// Rows sorted by expert: y[r] = act(x[src(r)] w[e(r)]^T), src(r) = sorted_src[r] / k (token of the route) or r itself.
// act: 0 none, 1 squared ReLU, 2 SiLU(gate) * up over weight rows that alternate (gate_i, up_i), y [rows, M / 2].
// Grid y counts 64-row tiles of all experts; a tile finds its expert by walking the offsets.
template <typename T>
__global__ void __launch_bounds__(256) expert_gemm_simt_kernel(const T* __restrict__ x, long long ldx, const int* __restrict__ sorted_src, int k, const T* __restrict__ w, T* __restrict__ y,
                                                               const int* __restrict__ offsets, int E, int M, int K, int act) {
  PG_PDL_ENTRY();
  __shared__ int s_e, s_row, s_end;
  if (threadIdx.x == 0) {
    int rem = blockIdx.y;
    s_e = -1;
    for (int e = 0; e < E; ++e) {
      const int a = offsets[e], b = offsets[e + 1], tiles = (b - a + 63) / 64;
      if (rem < tiles) {
        s_e = e, s_row = a + rem * 64, s_end = b;
        break;
      }
      rem -= tiles;
    }
  }
  __syncthreads();
  const int e = s_e;
  if (e < 0) return;
  const int m0 = blockIdx.x * 64, t0 = s_row, end = s_end;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  simt_tile(x, w + (long long)e * M * K, t0, end, m0, M, K, ldx, (long long)K, [=](int r) { return sorted_src ? sorted_src[r] / k : r; }, acc);
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, m = m0 + tx * 4 + j;
      if (t >= end || m >= M) continue;
      float v = acc[i][j];
      if (act == 2) {
        if (!(j & 1)) y[(long long)t * (M / 2) + m / 2] = from_f32<T>(glu_act(v, false) * acc[i][j | 1]);
        continue;
      }
      if (act == 1) v = v > 0.f ? v * v : 0.f;
      y[(long long)t * M + m] = from_f32<T>(v);
    }
}

constexpr int CONV_MAX = 16;   // taps
constexpr int CONV_TILE = 16;  // tokens per CTA; at least CONV_MAX - 1, so a sequence of more than one tile fills the carried inputs from its own rows

// A thread owns one channel for CONV_TILE tokens.  The CTA of a sequence's first tile reads the carried inputs and is also
// the one that replaces them (from the sequence's last rows), so no other CTA touches the state.
// CM: the number of taps rounded up to an instantiated size.  `bias` (or null) joins the sum, `in_bias` (or null) every input of
// the sequence, which is then rounded to T, as the carried ones are.
template <typename T, int CM>
__global__ void __launch_bounds__(128) short_conv_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ w, const float* __restrict__ bias, const float* __restrict__ in_bias, T* __restrict__ state,
                                                         T* __restrict__ out, long long ldo, const int* __restrict__ q_indptr, const int* __restrict__ slots, int channels, int taps, long long slot_stride, int silu) {
  PG_PDL_ENTRY();
  const int b = blockIdx.z, c = blockIdx.x * 128 + threadIdx.x;
  const int q0 = q_indptr[b], n = q_indptr[b + 1] - q0;
  const int s0 = blockIdx.y * CONV_TILE;
  const int slot = slots[b];
  if (c >= channels || s0 >= n || slot < 0) return;
  T* st = state + slot * slot_stride + (long long)c * (taps - 1);
  const int back = taps - 1;
  const int n_here = min(CONV_TILE, n - s0);
  const float cb = bias ? bias[c] : 0.f, ib = in_bias ? in_bias[c] : 0.f;
  auto input = [&](T v) { return in_bias ? from_f32<T>(to_f32(v) + ib) : v; };
  T rows[CONV_TILE];  // all loads of the tile in flight together
#pragma unroll
  for (int i = 0; i < CONV_TILE; ++i)
    if (i < n_here) rows[i] = x[(long long)(q0 + s0 + i) * ldx + c];
  // window and weights are right-aligned: entry CM - 1 belongs to the current row; inputs before this step come from the state
  float win[CM], wt[CM];
#pragma unroll
  for (int j = 0; j < CM; ++j) {
    const int tap = j - (CM - taps), at = s0 + j - (CM - 1);
    wt[j] = tap >= 0 ? w[(long long)c * taps + tap] : 0.f;
    win[j] = tap >= 0 && j < CM - 1 ? (at < 0 ? to_f32(st[back + at]) : to_f32(input(x[(long long)(q0 + at) * ldx + c]))) : 0.f;
  }
  T keep[CM];
  if (s0 == 0) {
#pragma unroll
    for (int j = 0; j < CM - 1; ++j) {
      const int at = n - back + j;
      if (j < back) keep[j] = at < 0 ? st[back + at] : input(x[(long long)(q0 + at) * ldx + c]);
    }
  }
#pragma unroll
  for (int i = 0; i < CONV_TILE; ++i) {
    if (i >= n_here) break;
    win[CM - 1] = to_f32(input(rows[i]));
    float a = cb;
#pragma unroll
    for (int j = 0; j < CM; ++j) a = fmaf(win[j], wt[j], a);
    out[(long long)(q0 + s0 + i) * ldo + c] = from_f32<T>(silu ? __fdividef(a, 1.f + __expf(-a)) : a);
#pragma unroll
    for (int j = 0; j < CM - 1; ++j) win[j] = win[j + 1];
  }
  if (s0 == 0) {
#pragma unroll
    for (int j = 0; j < CM - 1; ++j)
      if (j < back) st[j] = keep[j];
  }
}

inline bool al(const void* p, int bytes) { return ((uintptr_t)p % bytes) == 0; }

}  // namespace

// Element types of the calls below: 0 bf16, 1 f32.
extern "C" int pg_embed_rows(const void* table, int table_f32, long long ldt, const void* ids, void* x_f32, void* xt, int xt_f32, long long ldxt, int tokens, int width, long long rows, void* status, cudaStream_t stream) {
  if (tokens == 0) return PG_OK;
#define PG_EMBED(TI, TO) launch_pdl(embed_rows_kernel<TI, TO>, dim3(tokens), dim3(256), (size_t)0, stream, (const TI*)table, ldt, (const int*)ids, (float*)x_f32, (TO*)xt, ldxt, width, rows, (uint32_t*)status)
  if (table_f32)
    PG_CUDA(xt_f32 ? PG_EMBED(float, float) : PG_EMBED(float, bf16));
  else
    PG_CUDA(xt_f32 ? PG_EMBED(bf16, float) : PG_EMBED(bf16, bf16));
#undef PG_EMBED
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_post_norm(const void* y, int y_f32, long long ldy, const void* x_in, void* x_out, float alpha, const void* w, void* xt, int xt_f32, long long ldxt, int tokens, int width, float eps, cudaStream_t stream) {
  PG_REQUIRE(x_in != nullptr && w != nullptr && (x_out || xt), "post_norm: the stream, its norm weight and a destination are required");
  if (tokens == 0) return PG_OK;
  const int yb = y_f32 ? 4 : 2, tb = xt_f32 ? 4 : 2;
  const bool v4 = width % 4 == 0 && al(x_in, 16) && al(w, 16) && (!x_out || al(x_out, 16)) && (!y || (ldy % 4 == 0 && al(y, 4 * yb))) && (!xt || (ldxt % 4 == 0 && al(xt, 4 * tb)));
#define PG_PN(TY, TO, V) launch_pdl(post_norm_kernel<TY, TO, V>, dim3(tokens), dim3(256), (size_t)0, stream, (const TY*)y, ldy, (const float*)x_in, (float*)x_out, alpha, (const float*)w, (TO*)xt, ldxt, width, eps)
#define PG_PN2(TY, TO) (v4 ? PG_PN(TY, TO, 4) : PG_PN(TY, TO, 1))
  if (y_f32)
    PG_CUDA(xt_f32 ? PG_PN2(float, float) : PG_PN2(float, bf16));
  else
    PG_CUDA(xt_f32 ? PG_PN2(bf16, float) : PG_PN2(bf16, bf16));
#undef PG_PN2
#undef PG_PN
  PG_LAUNCH_CHECK();
  return PG_OK;
}

// table and pairs of one type; x f32 [tokens, width], xt [tokens, width]; carried int32 per slot: 1 + the previous token (0: none).
extern "C" int pg_embed_pairs_norm(const void* table, int table_f32, long long ldt, const void* pairs, long long ldp, const void* ids, const void* unit_seq, const void* q_indptr, const void* slots, void* carried,
                                   float scale, long long buckets, long long mul_prev, long long mul_cur, const void* w, void* x, void* xt, int xt_f32, int tokens, int width, long long rows, float eps,
                                   void* status, cudaStream_t stream) {
  PG_REQUIRE(pairs == nullptr || (buckets >= 1 && mul_prev >= 0 && mul_cur >= 0 && mul_prev < (1ll << 31) && mul_cur < (1ll << 31) && carried && unit_seq && q_indptr && slots),
             "embed_pairs: %lld buckets, multipliers %lld and %lld", buckets, mul_prev, mul_cur);
  if (tokens == 0) return PG_OK;
  const int ib = table_f32 ? 4 : 2, ob = xt_f32 ? 4 : 2;
  const bool v4 = width % 4 == 0 && al(table, 4 * ib) && ldt % 4 == 0 && (!pairs || (al(pairs, 4 * ib) && ldp % 4 == 0)) && al(w, 16) && al(x, 16) && al(xt, 4 * ob);
#define PG_EP(T, TO, V)                                                                                                                                                                            \
  launch_pdl(embed_pairs_norm_kernel<T, TO, V>, dim3(tokens), dim3(256), (size_t)0, stream, (const T*)table, ldt, (const T*)pairs, ldp, (const int*)ids, (const int*)unit_seq, (const int*)q_indptr, \
             (const int*)slots, (int*)carried, scale, buckets, mul_prev, mul_cur, (const float*)w, (float*)x, (TO*)xt, width, rows, eps, (uint32_t*)status)
#define PG_EP2(T, TO) (v4 ? PG_EP(T, TO, 4) : PG_EP(T, TO, 1))
  if (table_f32)
    PG_CUDA(xt_f32 ? PG_EP2(float, float) : PG_EP2(float, bf16));
  else
    PG_CUDA(xt_f32 ? PG_EP2(bf16, float) : PG_EP2(bf16, bf16));
#undef PG_EP2
#undef PG_EP
  PG_LAUNCH_CHECK();
  return PG_OK;
}

// y as in pg_add_layer_norm; extra (or null): a further row per token, times the sigmoid of extra_gate[token * ldg] (f32).
extern "C" int pg_residual_norm(const void* y, int y_f32, long long ldy, const void* pos, const void* weights, int k, const void* extra, int extra_f32, long long lde, const void* extra_gate, long long ldg,
                                void* x, float mult, const void* w, void* xt, int xt_f32, long long ldxt, int tokens, int width, float eps, cudaStream_t stream) {
  PG_REQUIRE(y != nullptr && w != nullptr && x != nullptr && xt != nullptr, "residual_norm: rows, the stream, the norm weight and a destination are required");
  PG_REQUIRE((pos == nullptr) == (weights == nullptr) && (pos == nullptr || k >= 1), "residual_norm: row positions and weights come together");
  if (tokens == 0) return PG_OK;
  const int yb = y_f32 ? 4 : 2, tb = xt_f32 ? 4 : 2, eb = extra_f32 ? 4 : 2;
  const bool v4 = width % 4 == 0 && al(w, 16) && al(x, 16) && ldy % 4 == 0 && al(y, 4 * yb) && ldxt % 4 == 0 && al(xt, 4 * tb) && (!extra || (lde % 4 == 0 && al(extra, 4 * eb)));
#define PG_RN(TY, TO, V)                                                                                                                                                                           \
  launch_pdl(residual_norm_kernel<TY, TO, V>, dim3(tokens), dim3(256), (size_t)0, stream, RowSource<TY>{(const TY*)y, ldy, (const int*)pos, (const float*)weights, k}, extra, extra_f32, lde,       \
             (const float*)extra_gate, ldg, (float*)x, mult, (const float*)w, (TO*)xt, ldxt, width, eps)
#define PG_RN2(TY, TO) (v4 ? PG_RN(TY, TO, 4) : PG_RN(TY, TO, 1))
  if (y_f32)
    PG_CUDA(xt_f32 ? PG_RN2(float, float) : PG_RN2(float, bf16));
  else
    PG_CUDA(xt_f32 ? PG_RN2(bf16, float) : PG_RN2(bf16, bf16));
#undef PG_RN2
#undef PG_RN
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_tanh_rows(const void* x, void* y, long long n, int is_f32, cudaStream_t stream) {
  if (n == 0) return PG_OK;
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  PG_CUDA(is_f32 ? launch_pdl(tanh_rows_kernel<float>, dim3((unsigned)blocks), dim3(256), (size_t)0, stream, (const float*)x, (float*)y, n)
                 : launch_pdl(tanh_rows_kernel<bf16>, dim3((unsigned)blocks), dim3(256), (size_t)0, stream, (const bf16*)x, (bf16*)y, n));
  PG_LAUNCH_CHECK();
  return PG_OK;
}

// y: [tokens, ldy] rows, or with pos / weights [tokens, k] the expert rows that pos points into (their weighted sum is the
// token's y).  x: f32 stream, updated in place (null: none, and then the norm itself goes to xt).
extern "C" int pg_add_layer_norm(const void* y, int y_f32, long long ldy, const void* pos, const void* weights, int k, void* x, const void* w, void* xt, int xt_f32, long long ldxt, int tokens, int width,
                                 float eps, cudaStream_t stream) {
  PG_REQUIRE(y != nullptr && w != nullptr && (x || xt), "add_layer_norm: rows, the norm weight and a destination are required");
  PG_REQUIRE((pos == nullptr) == (weights == nullptr) && (pos == nullptr || k >= 1), "add_layer_norm: row positions and weights come together");
  if (tokens == 0) return PG_OK;
  const int yb = y_f32 ? 4 : 2, tb = xt_f32 ? 4 : 2;
  const bool v4 = width % 4 == 0 && al(w, 16) && (!x || al(x, 16)) && ldy % 4 == 0 && al(y, 4 * yb) && (!xt || (ldxt % 4 == 0 && al(xt, 4 * tb)));
#define PG_LN(TY, TO, V)                                                                                                                                                                             \
  launch_pdl(add_layer_norm_kernel<TY, TO, V>, dim3(tokens), dim3(256), (size_t)0, stream, RowSource<TY>{(const TY*)y, ldy, (const int*)pos, (const float*)weights, k}, (float*)x, (const float*)w, \
             (TO*)xt, ldxt, width, eps)
#define PG_LN2(TY, TO) (v4 ? PG_LN(TY, TO, 4) : PG_LN(TY, TO, 1))
  if (y_f32)
    PG_CUDA(xt_f32 ? PG_LN2(float, float) : PG_LN2(float, bf16));
  else
    PG_CUDA(xt_f32 ? PG_LN2(bf16, float) : PG_LN2(bf16, bf16));
#undef PG_LN2
#undef PG_LN
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_gated_row_norm(const void* x, const void* gate, long long ldg, const void* w, void* y, int tokens, int heads, int dim, float eps, int silu, int w_heads, int gate_first,
                                 int is_f32, cudaStream_t stream) {
  if (tokens == 0) return PG_OK;
  const long long rows = (long long)tokens * heads;
  const bool wide = dim > 512;
  const bool v8 = !is_f32 && dim % 8 == 0 && ldg % 8 == 0 && al(x, 16) && al(gate, 16) && al(w, 16) && al(y, 16);
  const bool half = v8 && dim <= 128;  // a half warp covers the row with one access per lane
  const dim3 grid((unsigned)(wide ? rows : half ? (rows + 15) / 16 : (rows + 7) / 8));
#define PG_GRN(T, V, TPR) launch_pdl(gated_row_norm_kernel<T, V, TPR>, grid, dim3(256), (size_t)0, stream, (const T*)x, (const T*)gate, ldg, (const float*)w, (T*)y, rows, heads, dim, eps, silu, w_heads, gate_first)
  if (is_f32) {
    PG_CUDA(wide ? PG_GRN(float, 1, 256) : PG_GRN(float, 1, 32));
  } else {
    if (v8)
      PG_CUDA(wide ? PG_GRN(bf16, 8, 256) : half ? PG_GRN(bf16, 8, 16) : PG_GRN(bf16, 8, 32));
    else
      PG_CUDA(wide ? PG_GRN(bf16, 1, 256) : PG_GRN(bf16, 1, 32));
  }
#undef PG_GRN
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_glu_rows_f32(const void* gu, void* out, int rows, int inter, long long ldin, int gelu, cudaStream_t stream) {
  if (rows == 0 || inter == 0) return PG_OK;
  long long blocks = ((long long)rows * inter + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  PG_CUDA(launch_pdl(glu_rows_kernel, dim3((unsigned)blocks), dim3(256), (size_t)0, stream, (const float*)gu, (float*)out, rows, inter, ldin, gelu));
  PG_LAUNCH_CHECK();
  return PG_OK;
}

// x f32, y f32 or bf16; act: f32 softplus(p), 1/2 + softplus(q).
extern "C" int pg_xielu_rows(const void* x, void* y, const void* act, long long n, int y_f32, cudaStream_t stream) {
  if (n == 0) return PG_OK;
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  PG_CUDA(y_f32 ? launch_pdl(xielu_rows_kernel<float>, dim3((unsigned)blocks), dim3(256), (size_t)0, stream, (const float*)x, (float*)y, (const float*)act, n)
                : launch_pdl(xielu_rows_kernel<bf16>, dim3((unsigned)blocks), dim3(256), (size_t)0, stream, (const float*)x, (bf16*)y, (const float*)act, n));
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_softcap_f32(const void* x, void* y, long long n, float cap, cudaStream_t stream) {
  PG_REQUIRE(cap > 0.f, "softcap: the cap must be positive");
  if (n == 0) return PG_OK;
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  PG_CUDA(launch_pdl(softcap_f32_kernel, dim3((unsigned)blocks), dim3(256), (size_t)0, stream, (const float*)x, (float*)y, n, cap));
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_gemm_simt(const void* x, const void* w, int x_f32, void* y, int y_f32, int T, int M, int K, long long ldx, long long ldw, long long ldy, cudaStream_t stream) {
  PG_REQUIRE(T > 0 && M > 0 && K > 0, "gemm_simt: empty problem %dx%dx%d", T, M, K);
  const dim3 grid((M + 63) / 64, (T + 63) / 64);
  PG_REQUIRE(grid.y <= 65535u, "gemm_simt: %d rows", T);
#define PG_SG(TX, TY) launch_pdl(gemm_simt_kernel<TX, TY>, grid, dim3(256), (size_t)0, stream, (const TX*)x, (const TX*)w, (TY*)y, T, M, K, ldx, ldw, ldy)
  if (x_f32)
    PG_CUDA(y_f32 ? PG_SG(float, float) : PG_SG(float, bf16));
  else
    PG_CUDA(y_f32 ? PG_SG(bf16, float) : PG_SG(bf16, bf16));
#undef PG_SG
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_head_gemm_simt(const void* x, long long ldx, long long x_head, const void* w, void* y, long long ldy, long long y_head, const void* gate, long long ldg, long long g_head, int heads,
                                 int rows, int M, int K, int y_f32, int is_f32, cudaStream_t stream) {
  PG_REQUIRE(heads > 0 && rows > 0 && M > 0 && K > 0, "head_gemm_simt: empty problem");
  const dim3 grid((M + 63) / 64, (rows + 63) / 64, heads);
  PG_REQUIRE(grid.y <= 65535u && grid.z <= 65535u, "head_gemm_simt: %d rows of %d heads", rows, heads);
#define PG_HG(T, TY) launch_pdl(head_gemm_simt_kernel<T, TY>, grid, dim3(256), (size_t)0, stream, (const T*)x, ldx, x_head, (const T*)w, (TY*)y, ldy, y_head, (const T*)gate, ldg, g_head, rows, M, K)
  PG_REQUIRE(y_f32 || !is_f32, "head_gemm_simt: f32 operands give f32");
  PG_CUDA(is_f32 ? PG_HG(float, float) : y_f32 ? PG_HG(bf16, float) : PG_HG(bf16, bf16));
#undef PG_HG
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_expert_gemm_simt(const void* x, long long ldx, const void* sorted_src, int k, const void* w, void* y, const void* offsets, int routes, int E, int M, int K, int act, int is_f32,
                                   cudaStream_t stream) {
  PG_REQUIRE(act != 2 || M % 2 == 0, "expert_gemm_simt: %d rows are not pairs of gate and up", M);
  if (routes == 0) return PG_OK;
  const dim3 grid((M + 63) / 64, (routes + 63) / 64 + (E < routes ? E : routes));
  PG_REQUIRE(M > 0 && K > 0 && grid.y <= 65535u, "expert_gemm_simt: %d routes, %d x %d", routes, M, K);
#define PG_EG(T) launch_pdl(expert_gemm_simt_kernel<T>, grid, dim3(256), (size_t)0, stream, (const T*)x, ldx, (const int*)sorted_src, k, (const T*)w, (T*)y, (const int*)offsets, E, M, K, act)
  PG_CUDA(is_f32 ? PG_EG(float) : PG_EG(bf16));
#undef PG_EG
  PG_LAUNCH_CHECK();
  return PG_OK;
}

// bias, in_bias: f32 [channels] or null; silu: the activation of the sum.
extern "C" int pg_short_conv(const void* x, long long ldx, const void* w, const void* bias, const void* in_bias, void* state, void* out, long long ldo, const void* q_indptr, const void* slots, int num_seqs, int channels,
                             int taps, long long slot_stride, int max_q_len, int silu, int is_f32, cudaStream_t stream) {
  PG_REQUIRE(taps >= 1 && taps <= CONV_MAX, "short_conv: %d taps (1..%d)", taps, CONV_MAX);
  if (num_seqs == 0) return PG_OK;
  const dim3 grid((channels + 127) / 128, (max_q_len + CONV_TILE - 1) / CONV_TILE, num_seqs);
  PG_REQUIRE(grid.y <= 65535u && grid.z <= 65535u, "short_conv: %d sequences of %d rows", num_seqs, max_q_len);
#define PG_CONV(T, CM) launch_pdl(short_conv_kernel<T, CM>, grid, dim3(128), (size_t)0, stream, (const T*)x, ldx, (const float*)w, (const float*)bias, (const float*)in_bias, (T*)state, (T*)out, ldo, (const int*)q_indptr, (const int*)slots, channels, taps, slot_stride, silu)
#define PG_CONVS(T) (taps <= 2 ? PG_CONV(T, 2) : taps <= 4 ? PG_CONV(T, 4) : taps <= 8 ? PG_CONV(T, 8) : PG_CONV(T, 16))
  PG_CUDA(is_f32 ? PG_CONVS(float) : PG_CONVS(bf16));
#undef PG_CONVS
#undef PG_CONV
  PG_LAUNCH_CHECK();
  return PG_OK;
}
