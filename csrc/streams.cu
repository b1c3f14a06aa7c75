// Row kernels of a residual stream that is kept in several copies (hyper-connections), all in 32 bits.
//
//  * embed_positions: table row plus the sinusoids of the token's position, whose angle is the sum of a coarse and a fine part
//    (sin(a + b) and cos(a + b) from two small tables, so that no table has a row per position).
//  * streams_norm: everything between two sublayers in one pass over the copies x[0 .. s) of a token.
//      x'[t] = sum_s mix[s, t] x[s] + out[t] y          (y: the sublayer's output)
//      u     = sum_s old[s] x[s] + new y                (the next sublayer's input, sum_t gather[t] x'[t] with the sums folded)
//      h     = u / sqrt(mean(u^2) + eps) * w
//    and, in front of a mixer with a token shift, h + (h_prev - h) * shift with the previous token's h.
//    A CTA takes `run` consecutive rows, so the previous row's h is usually still in its registers.  In front of a run it is formed
//    once more from the old copies (the new ones go to another buffer, so nobody overwrites them); in front of a sequence it comes
//    from the request's slot.  The CTA of a sequence's first row is the only one that touches the slot: it also puts the h of the
//    sequence's last row there.
#include "api.h"
#include "common.cuh"
#include "types.cuh"

namespace {

constexpr int FINE = 256;  // positions of the fine table

template <typename T>
__global__ void __launch_bounds__(256) embed_positions_kernel(const T* __restrict__ table, long long ldt, const float2* __restrict__ coarse, const float2* __restrict__ fine, const int* __restrict__ ids,
                                                              const int* __restrict__ positions, float* __restrict__ x, int width, long long rows, int coarse_rows, uint32_t* status) {
  PG_PDL_ENTRY();
  const long long t = blockIdx.x;
  long long id = ids[t];
  int pos = positions[t];
  if (id < 0 || id >= rows || pos < 0 || pos >= coarse_rows * FINE) {
    if (threadIdx.x == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (59u << 8));
    id = 0, pos = 0;
  }
  const int pairs = (width + 1) / 2;
  const float2 *a = coarse + (long long)(pos / FINE) * pairs, *b = fine + (long long)(pos % FINE) * pairs;
  for (int i = threadIdx.x; i < pairs; i += 256) {
    const float2 p = a[i], q = b[i];  // (sine, cosine)
    x[t * width + 2 * i] = to_f32(table[id * ldt + 2 * i]) + (p.x * q.y + p.y * q.x);
    if (2 * i + 1 < width) x[t * width + 2 * i + 1] = to_f32(table[id * ldt + 2 * i + 1]) + (p.y * q.y - p.x * q.x);
  }
}

struct StreamArgs {
  const float* x;  // [tokens, s_in, width]
  int s_in;
  const void* y;  // [tokens, width] rows of stride ldy, or null
  long long ldy;
  const float* coef;  // mix [s_in, s_out] | out [s_out] | old [s_in] | new
  float* x_out;       // [tokens, s_out, width], or null
  int s_out;
  const float* w;
  void* h;  // [tokens, width]
  const float* shift;
  float* carried;  // [slots, width]
  const int *unit_seq, *q_indptr, *slots;
  int tokens, width, run;
  float eps;
};

// S: copies rounded up to an instantiated size, a token's copies and the coefficients in registers; 0: any number, both read where they
// are used.  A thread owns up to KEEP vectors of V columns.
template <typename TY, typename TO, int S, int V, int KEEP>
__global__ void __launch_bounds__(512) streams_norm_kernel(const StreamArgs p) {
  PG_PDL_ENTRY();
  __shared__ float red[32];
  const int width = p.width, nv = width / V, threads = blockDim.x;
  const TY* y = reinterpret_cast<const TY*>(p.y);
  TO* hout = reinterpret_cast<TO*>(p.h);
  const bool keep = p.x_out != nullptr, add = y != nullptr;
  const float *c_out = p.coef + p.s_in * p.s_out, *c_old = c_out + p.s_out;
  const float c_new = c_old[p.s_in];
  constexpr int R = S > 0 ? S : 1;
  float mix[R][R], out[R], old[R];
  if constexpr (S > 0) {
#pragma unroll
    for (int s = 0; s < S; ++s) {
      old[s] = s < p.s_in ? c_old[s] : 0.f;
      out[s] = s < p.s_out ? c_out[s] : 0.f;
#pragma unroll
      for (int t = 0; t < S; ++t) mix[s][t] = s < p.s_in && t < p.s_out ? p.coef[s * p.s_out + t] : 0.f;
    }
  }

  // normed row t (without the token shift) in h; `store`: its new copies go out
  auto row = [&](long long t, bool store, float (&h)[KEEP][V]) {
    const float* xr = p.x + t * p.s_in * width;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = threadIdx.x + k * threads;
      if (i >= nv) continue;
      float x[R][V], yv[V];
#pragma unroll
      for (int s = 0; s < S; ++s)
        if (s < p.s_in) load_vec<V>(xr + (long long)s * width + i * V, x[s]);
#pragma unroll
      for (int j = 0; j < V; ++j) yv[j] = 0.f;
      if (add) load_vec<V>(y + t * p.ldy + i * V, yv);
      if constexpr (S == 0) {
        auto sum = [&](float first, const float* c, int step, float (&o)[V]) {  // first * y + sum_s c[s * step] x[s]
#pragma unroll
          for (int j = 0; j < V; ++j) o[j] = first * yv[j];
#pragma unroll 1
          for (int s = 0; s < p.s_in; ++s) {
            load_vec<V>(xr + (long long)s * width + i * V, x[0]);
#pragma unroll
            for (int j = 0; j < V; ++j) o[j] = fmaf(c[s * step], x[0][j], o[j]);
          }
        };
        sum(c_new, c_old, 1, h[k]);
#pragma unroll
        for (int j = 0; j < V; ++j) ss += h[k][j] * h[k][j];
        if (keep && store) {
#pragma unroll 1
          for (int n = 0; n < p.s_out; ++n) {
            float o[V];
            sum(c_out[n], p.coef + n, p.s_out, o);
            store_vec<V>(p.x_out + (t * p.s_out + n) * width + i * V, o);
          }
        }
        continue;
      }
#pragma unroll
      for (int j = 0; j < V; ++j) {
        float u = c_new * yv[j];
#pragma unroll
        for (int s = 0; s < S; ++s)
          if (s < p.s_in) u = fmaf(old[s], x[s][j], u);
        h[k][j] = u;
        ss += u * u;
      }
      if (keep && store) {
#pragma unroll
        for (int n = 0; n < S; ++n)
          if (n < p.s_out) {
            float o[V];
#pragma unroll
            for (int j = 0; j < V; ++j) {
              o[j] = out[n] * yv[j];
#pragma unroll
              for (int s = 0; s < S; ++s)
                if (s < p.s_in) o[j] = fmaf(mix[s][n], x[s][j], o[j]);
            }
            store_vec<V>(p.x_out + (t * p.s_out + n) * width + i * V, o);
          }
      }
    }
    const float inv = rsqrtf(block_sum(ss, red) / (float)width + p.eps);
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = threadIdx.x + k * threads;
      if (i >= nv) continue;
      float wf[V];
      load_vec<V>(p.w + i * V, wf);
#pragma unroll
      for (int j = 0; j < V; ++j) h[k][j] *= inv * wf[j];
    }
  };

  const int t0 = blockIdx.x * p.run, t1 = min(p.tokens, t0 + p.run);
  float h[KEEP][V], back[KEEP][V];
  for (int t = t0; t < t1; ++t) {
    row(t, true, h);
    if (p.shift) {
      const int b = p.unit_seq[t];
      if (t == p.q_indptr[b]) {
        const int slot = p.slots[b], last = p.q_indptr[b + 1] - 1;
        float* st = p.carried + (long long)(slot < 0 ? 0 : slot) * width;
        float end[KEEP][V];
        if (slot >= 0 && last != t) row(last, false, end);
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
          const int i = threadIdx.x + k * threads;
          if (i >= nv) continue;
          if (slot >= 0) {
            load_vec<V>(st + i * V, back[k]);
            store_vec<V>(st + i * V, last != t ? end[k] : h[k]);
          } else {
#pragma unroll
            for (int j = 0; j < V; ++j) back[k][j] = 0.f;
          }
        }
      } else if (t == t0) {
        row(t - 1, false, back);
      }
    }
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = threadIdx.x + k * threads;
      if (i >= nv) continue;
      float o[V];
      if (p.shift) {
        float m[V];
        load_vec<V>(p.shift + i * V, m);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          o[j] = fmaf(back[k][j] - h[k][j], m[j], h[k][j]);
          back[k][j] = h[k][j];
        }
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) o[j] = h[k][j];
      }
      store_vec<V>(hout + (long long)t * width + i * V, o);
    }
  }
}

inline bool al(const void* p, int bytes) { return ((uintptr_t)p % bytes) == 0; }

template <typename TY, typename TO, int S, int V, int KEEP>
cudaError_t launch_streams(const StreamArgs& p, int threads, cudaStream_t stream) {
  return launch_pdl(streams_norm_kernel<TY, TO, S, V, KEEP>, dim3((p.tokens + p.run - 1) / p.run), dim3(threads), (size_t)0, stream, p);
}
template <typename TY, typename TO, int V, int KEEP>
cudaError_t launch_copies(const StreamArgs& p, int threads, cudaStream_t stream) {
  const int s = p.s_in > p.s_out ? p.s_in : p.s_out;
  if (s <= 2) return launch_streams<TY, TO, 2, V, KEEP>(p, threads, stream);
  if (s <= 4) return launch_streams<TY, TO, 4, V, KEEP>(p, threads, stream);
  return launch_streams<TY, TO, 0, V, KEEP>(p, threads, stream);
}
template <typename TY, typename TO>
cudaError_t launch_rows(const StreamArgs& p, bool v4, cudaStream_t stream) {
  const int nv = p.width / (v4 ? 4 : 1);
  auto threads = [&](int per) { return ((nv + per - 1) / per + 31) / 32 * 32; };
  // few rows: up to 512 threads per row; many rows: four vectors per thread, so that several rows are in flight per SM
  if (v4 && nv <= 1024 && p.tokens < 2 * 148) return launch_copies<TY, TO, 4, 2>(p, threads(nv <= 512 ? 1 : 2), stream);
  if (v4) return launch_copies<TY, TO, 4, 4>(p, threads(4), stream);
  return launch_copies<TY, TO, 1, 8>(p, threads(8), stream);
}

}  // namespace

// table [rows, width] of one type (table_f32: f32, else bf16); coarse f32 [coarse_rows, pairs, 2], fine f32 [256, pairs, 2]; x f32 [tokens, width].
extern "C" int pg_embed_positions(const void* table, int table_f32, long long ldt, const void* coarse, int coarse_rows, const void* fine, const void* ids, const void* positions, void* x, int tokens, int width,
                                  long long rows, void* status, cudaStream_t stream) {
  PG_REQUIRE(width >= 1 && coarse_rows >= 1 && rows >= 1, "embed_positions: %d columns, %d coarse rows", width, coarse_rows);
  if (tokens == 0) return PG_OK;
#define PG_EPO(T)                                                                                                                                                                              \
  launch_pdl(embed_positions_kernel<T>, dim3(tokens), dim3(256), (size_t)0, stream, (const T*)table, ldt, (const float2*)coarse, (const float2*)fine, (const int*)ids, (const int*)positions, \
             (float*)x, width, rows, coarse_rows, (uint32_t*)status)
  PG_CUDA(table_f32 ? PG_EPO(float) : PG_EPO(bf16));
#undef PG_EPO
  PG_LAUNCH_CHECK();
  return PG_OK;
}

// x f32 [tokens, s_in, width]; y (bf16 or f32 rows of stride ldy, or null); coef as in StreamArgs; x_out f32 [tokens, s_out, width] or null (another
// buffer than x); h [tokens, width] in the activation type; shift f32 [width] or null, and with it carried f32 [slots, width], the sequence of
// every row, the first rows of the sequences and their slots.
extern "C" int pg_streams_norm(const void* x, int s_in, const void* y, int y_f32, long long ldy, const void* coef, void* x_out, int s_out, const void* w, void* h, int h_f32, const void* shift, void* carried,
                               const void* unit_seq, const void* q_indptr, const void* slots, int tokens, int width, float eps, cudaStream_t stream) {
  PG_REQUIRE(s_in >= 1 && s_out >= 1, "streams_norm: %d copies to %d", s_in, s_out);
  PG_REQUIRE(x && coef && w && h && x != x_out && (shift == nullptr || (carried && unit_seq && q_indptr && slots)), "streams_norm: an operand is missing, or the copies would be overwritten");
  if (tokens == 0) return PG_OK;
  StreamArgs p = {(const float*)x, s_in, y, ldy, (const float*)coef, (float*)x_out, s_out, (const float*)w, h, (const float*)shift, (float*)carried, (const int*)unit_seq, (const int*)q_indptr,
                  (const int*)slots, tokens, width, 1, eps};
  const int yb = y_f32 ? 4 : 2, hb = h_f32 ? 4 : 2;
  const bool v4 = width % 4 == 0 && al(x, 16) && (!y || (al(y, 4 * yb) && ldy % 4 == 0)) && (!x_out || al(x_out, 16)) && al(w, 16) && al(h, 4 * hb) && (!shift || (al(shift, 16) && al(carried, 16)));
  PG_REQUIRE(width / (v4 ? 4 : 1) <= (v4 ? 2048 : 4096), "streams_norm: rows of %d columns", width);
  if (shift)  // with a token shift a run of rows saves forming the row in front of it once more
    while (p.run < 16 && (tokens + 2 * p.run - 1) / (2 * p.run) >= 148 * 4) p.run *= 2;
  if (y_f32 || !y)
    PG_CUDA(h_f32 ? (launch_rows<float, float>(p, v4, stream)) : (launch_rows<float, bf16>(p, v4, stream)));
  else
    PG_CUDA(h_f32 ? (launch_rows<bf16, float>(p, v4, stream)) : (launch_rows<bf16, bf16>(p, v4, stream)));
  PG_LAUNCH_CHECK();
  return PG_OK;
}
