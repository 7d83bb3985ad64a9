// Typed loads and stores for kernels that exist for bf16 and fp32 activations: everything is computed in fp32,
// the template argument only says how a tensor is stored.
#pragma once

#include "tw_common.cuh"

namespace tw {

// Storage types of the `dtype` argument of the launchers.
enum : int { TW_BF16 = 0, TW_F32 = 1 };

__device__ __forceinline__ float ld1(const float* p) { return *p; }
__device__ __forceinline__ float ld1(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st1(float* p, float v) { *p = v; }
__device__ __forceinline__ void st1(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// Eight consecutive elements (16-byte aligned rows).
__device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void ld8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y), c = unpack_bf16x2(u.z), d = unpack_bf16x2(u.w);
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  v[4] = c.x; v[5] = c.y; v[6] = d.x; v[7] = d.y;
}
__device__ __forceinline__ void st8(float* p, const float (&v)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void st8(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 u;
  u.x = pack_bf16x2(v[0], v[1]);
  u.y = pack_bf16x2(v[2], v[3]);
  u.z = pack_bf16x2(v[4], v[5]);
  u.w = pack_bf16x2(v[6], v[7]);
  *reinterpret_cast<uint4*>(p) = u;
}

// Eight consecutive elements of which the first `n` are inside the row; VEC: rows are 16-byte aligned and a
// full group is one vector access.
template <bool VEC, typename T>
__device__ __forceinline__ void ld8n(const T* p, int n, float (&v)[8]) {
  if (VEC && n >= 8) {
    ld8(p, v);
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = j < n ? ld1(p + j) : 0.f;
  }
}
template <bool VEC, typename T>
__device__ __forceinline__ void st8n(T* p, int n, const float (&v)[8]) {
  if (VEC && n >= 8) {
    st8(p, v);
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (j < n) st1(p + j, v[j]);
  }
}

// Eight elements as they are stored (a request whose conversion can wait).
template <typename T>
struct __align__(16) Raw8 {
  T v[8];
};
template <bool VEC, typename T>
__device__ __forceinline__ Raw8<T> ld8raw(const T* p, int n) {
  Raw8<T> r;
  if (VEC && n >= 8) {
    if constexpr (sizeof(T) == 2) {
      *reinterpret_cast<uint4*>(&r) = *reinterpret_cast<const uint4*>(p);
    } else {
      reinterpret_cast<uint4*>(&r)[0] = reinterpret_cast<const uint4*>(p)[0];
      reinterpret_cast<uint4*>(&r)[1] = reinterpret_cast<const uint4*>(p)[1];
    }
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) st1(&r.v[j], j < n ? ld1(p + j) : 0.f);
  }
  return r;
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
// Activations of bf16 tensors: the result is rounded to 8 bits of mantissa, the hardware exponential and division
// (__expf, __fdividef) are exact enough; fp32 tensors take the functions above.
template <typename T>
__device__ __forceinline__ float silu_t(float x) {
  if (sizeof(T) == 2) return __fdividef(x, 1.f + __expf(-x));
  return silu_f(x);
}
template <typename T>
__device__ __forceinline__ float sigmoid_t(float x) {
  if (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-x));
  return sigmoid_f(x);
}
// the tanh form of gelu, z / 2 (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3)))
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// -ln(decay) of a fixed decay per token; a decay of (nearly) nothing is kept finite, since differences of its multiples
// are formed (1e-30 wipes a state out in one token).
__device__ __forceinline__ double decay_rate(float decay) { return -log(static_cast<double>(fmaxf(decay, 1e-30f))); }

}  // namespace tw
