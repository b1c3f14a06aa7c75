// Element access for kernels that are instantiated for bf16 and f32 activations, and the hyperbolic tangent that the
// soft caps use (32-bit accuracy, whatever the fast-math flags make of tanhf).
#pragma once
#include "common.cuh"

#ifdef __CUDACC__

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16(v); }

// V elements with one access (V * sizeof(T) bytes, aligned) when V > 1
template <int V>
__device__ __forceinline__ void load_vec(const float* p, float* f) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V / 4; ++i) {
      const float4 t = reinterpret_cast<const float4*>(p)[i];
      f[4 * i] = t.x, f[4 * i + 1] = t.y, f[4 * i + 2] = t.z, f[4 * i + 3] = t.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = p[i];
  }
}
template <int V>
__device__ __forceinline__ void load_vec(const bf16* p, float* f) {
  if constexpr (V == 8) {
    unpack8(*reinterpret_cast<const bf16x8*>(p), f);
  } else if constexpr (V == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&t.x)), b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&t.y));
    f[0] = a.x, f[1] = a.y, f[2] = b.x, f[3] = b.y;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = __bfloat162float(p[i]);
  }
}
template <int V>
__device__ __forceinline__ void store_vec(float* p, const float* f) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V / 4; ++i) reinterpret_cast<float4*>(p)[i] = make_float4(f[4 * i], f[4 * i + 1], f[4 * i + 2], f[4 * i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = f[i];
  }
}
template <int V>
__device__ __forceinline__ void store_vec(bf16* p, const float* f) {
  if constexpr (V == 8) {
    *reinterpret_cast<bf16x8*>(p) = pack8(f);
  } else if constexpr (V == 4) {
    const bf162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    uint2 t;
    t.x = *reinterpret_cast<const uint32_t*>(&a), t.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = t;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = __float2bfloat16(f[i]);
  }
}

// tanh(x): the Taylor polynomial through x^11 below 0.3 (truncation under 1e-8 relative), (e^2x - 1) / (e^2x + 1) above.
__device__ __forceinline__ float tanh_full(float x) {
  const float a = fabsf(x), x2 = x * x;
  if (a < 0.3f)
    return x * (1.f + x2 * (-1.f / 3.f + x2 * (2.f / 15.f + x2 * (-17.f / 315.f + x2 * (62.f / 2835.f + x2 * (-1382.f / 155925.f))))));
  return copysignf(1.f - 2.f / (1.f + __expf(2.f * a)), x);
}

#endif  // __CUDACC__
