// Decays and element access shared by the kernels of input-dependent recurrences.
#pragma once

#include "xpool/elem.cuh"

namespace xpool {
namespace recur {

constexpr float kUnitEps = 1e-6f;          // added to a query's or key's sum of squares before it becomes a unit vector

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// log of sigmoid(z) ** inv_tau
__device__ __forceinline__ float log_decay(float z, float inv_tau) { return -softplus(-z) * inv_tau; }
__device__ __forceinline__ float delta_log_decay(float x, float neg_a, float dt_bias) { return neg_a * softplus(x + dt_bias); }

// VEC consecutive elements of 16 bytes (or one element).
template <int VEC>
__device__ __forceinline__ void ldx(const float* p, float (&x)[VEC]) {
  elem::ldv<VEC>(p, x);
}
template <int VEC>
__device__ __forceinline__ void ldx(const __nv_bfloat16* p, float (&x)[VEC]) {
  if constexpr (VEC == 8) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
      x[2 * i] = f.x, x[2 * i + 1] = f.y;
    }
  } else {
    x[0] = __bfloat162float(*p);
  }
}
template <int VEC, typename T>
__device__ __forceinline__ void ldr(const T* p, T (&x)[VEC]) {
  if constexpr (VEC * sizeof(T) == 16) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const T* e = reinterpret_cast<const T*>(&v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] = e[i];
  } else {
    x[0] = p[0];
  }
}
template <int VEC, typename T>
__device__ __forceinline__ void stx(T* p, const T (&x)[VEC]) {
  if constexpr (VEC * sizeof(T) == 16) {
    uint4 v;
    T* e = reinterpret_cast<T*>(&v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) e[i] = x[i];
    *reinterpret_cast<uint4*>(p) = v;
  } else {
    p[0] = x[0];
  }
}

}  // namespace recur
}  // namespace xpool
