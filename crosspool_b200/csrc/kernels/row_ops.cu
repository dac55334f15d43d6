// Row-wise kernels of layered decoders, one CTA per token row, everything computed in fp32:
//   resid_norm   [embedding gather | residual += sublayer output * sigmoid(gate)] -> norm -> activation row
//   polynorm     a N(z) + b N(z^2) + c N(z^3) + e, N dividing the row by its root mean square
//   gated_rms    rmsnorm(o) * w * sigmoid(gate)
// Rows whose pitches allow it are moved four elements at a time.
#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"

namespace xpool {
namespace rowops {

using elem::block_sum;
using elem::ldv;
using elem::sigmoid;
using elem::stv;

constexpr int kThreads = 256;
enum NormKind : int { kRms = 0, kLayer = 1, kDynTanh = 2 };

template <typename T, int N, int KIND>
__global__ void __launch_bounds__(kThreads)
resid_norm_kernel(XpResidNormArgs a) {
  __shared__ float red[kThreads / 32];
  const int i = blockIdx.x;
  const int r = a.sel != nullptr ? a.sel[i] : i;
  float* resid = a.resid + static_cast<size_t>(r) * a.hidden;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<size_t>(i) * a.ld_out;
  const T* gate = a.gate != nullptr ? reinterpret_cast<const T*>(a.gate) + static_cast<size_t>(r) * a.ld_gate : nullptr;
  const T* emb = nullptr;
  if (a.ids != nullptr) {
    int id = a.ids[r];
    if (id < 0 || id >= a.vocab) id = 0;
    emb = reinterpret_cast<const T*>(a.table) + static_cast<size_t>(id) * a.hidden;
  }
  const bool write_back = a.sel == nullptr && (emb != nullptr || a.nparts > 0);
  const float alpha = KIND == kDynTanh && a.out != nullptr ? *a.alpha : 0.f;

  auto residual = [&](int c, float (&v)[N]) {
    if (emb != nullptr) {
      ldv<N>(emb + c, v);
      return;
    }
    ldv<N>(resid + c, v);
    if (a.nparts == 0) return;
    float y[N];
#pragma unroll
    for (int j = 0; j < N; ++j) y[j] = 0.f;
    for (int p = 0; p < a.nparts; ++p) {
      float t[N];
      ldv<N>(reinterpret_cast<const T*>(a.parts[p]) + static_cast<size_t>(r) * a.ld_part + c, t);
#pragma unroll
      for (int j = 0; j < N; ++j) y[j] += t[j];
    }
    if (gate != nullptr) {
      float g[N];
      ldv<N>(gate + c, g);
#pragma unroll
      for (int j = 0; j < N; ++j) y[j] *= sigmoid(g[j]);
    }
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] += y[j];
  };
  auto finish = [&](int c, float (&v)[N], float mean, float inv) {
    float w[N], b[N];
    ldv<N>(a.weight + c, w);
#pragma unroll
    for (int j = 0; j < N; ++j) b[j] = 0.f;
    if (a.bias != nullptr) ldv<N>(a.bias + c, b);
#pragma unroll
    for (int j = 0; j < N; ++j) {
      const float n = KIND == kDynTanh ? tanhf(alpha * v[j]) : (v[j] - mean) * inv;
      v[j] = n * w[j] + b[j];
    }
    stv<N>(out + c, v);
  };

  float s1 = 0.f, s2 = 0.f;
  for (int c = threadIdx.x * N; c < a.hidden; c += kThreads * N) {
    float v[N];
    residual(c, v);
    if (write_back) stv<N>(resid + c, v);
    if (a.out == nullptr) continue;
    if constexpr (KIND == kDynTanh) {
      finish(c, v, 0.f, 0.f);
    } else {
#pragma unroll
      for (int j = 0; j < N; ++j) s1 += v[j], s2 += v[j] * v[j];
    }
  }
  if (KIND == kDynTanh || a.out == nullptr) return;
  const float n = static_cast<float>(a.hidden);
  float mean = 0.f;
  if constexpr (KIND == kLayer) {
    mean = block_sum<kThreads>(s1, red) / n;
    s2 = 0.f;
    for (int c = threadIdx.x * N; c < a.hidden; c += kThreads * N) {
      float v[N];
      if (write_back) ldv<N>(resid + c, v);
      else residual(c, v);
#pragma unroll
      for (int j = 0; j < N; ++j) s2 += (v[j] - mean) * (v[j] - mean);
    }
  }
  const float inv = rsqrtf(block_sum<kThreads>(s2, red) / n + a.eps);
  for (int c = threadIdx.x * N; c < a.hidden; c += kThreads * N) {
    float v[N];
    if (write_back) ldv<N>(resid + c, v);   // this thread's own store
    else residual(c, v);
    finish(c, v, mean, inv);
  }
}

// Values stay in registers between the two passes while a row has at most kThreads * kKeep elements.
constexpr int kKeep = 32;

template <typename T, int N>
__global__ void __launch_bounds__(kThreads)
polynorm_kernel(XpPolyNormArgs a) {
  __shared__ float red[kThreads / 32];
  const T* z = reinterpret_cast<const T*>(a.z) + static_cast<size_t>(blockIdx.x) * a.ld_z;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<size_t>(blockIdx.x) * a.ld_out;
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  float keep[kKeep / N][N];
#pragma unroll
  for (int it = 0; it < kKeep / N; ++it) {
    const int c = (it * kThreads + threadIdx.x) * N;
    if (c < a.cols) {
      ldv<N>(z + c, keep[it]);
#pragma unroll
      for (int j = 0; j < N; ++j) {
        const float q = keep[it][j] * keep[it][j];
        s1 += q, s2 += q * q, s3 += q * q * q;
      }
    }
  }
  for (int c = (kKeep / N * kThreads + threadIdx.x) * N; c < a.cols; c += kThreads * N) {
    float v[N];
    ldv<N>(z + c, v);
#pragma unroll
    for (int j = 0; j < N; ++j) {
      const float q = v[j] * v[j];
      s1 += q, s2 += q * q, s3 += q * q * q;
    }
  }
  const float n = static_cast<float>(a.cols);
  const float c1 = a.coef[0] * rsqrtf(block_sum<kThreads>(s1, red) / n + a.eps);
  const float c2 = a.coef[1] * rsqrtf(block_sum<kThreads>(s2, red) / n + a.eps);
  const float c3 = a.coef[2] * rsqrtf(block_sum<kThreads>(s3, red) / n + a.eps);
  const float c0 = a.coef[3];
  auto store = [&](int c, float (&v)[N]) {
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = fmaf(fmaf(fmaf(c3, v[j], c2), v[j], c1), v[j], c0);
    stv<N>(out + c, v);
  };
#pragma unroll
  for (int it = 0; it < kKeep / N; ++it) {
    const int c = (it * kThreads + threadIdx.x) * N;
    if (c < a.cols) store(c, keep[it]);
  }
  for (int c = (kKeep / N * kThreads + threadIdx.x) * N; c < a.cols; c += kThreads * N) {
    float v[N];
    ldv<N>(z + c, v);
    store(c, v);
  }
}

template <typename T, int N>
__global__ void __launch_bounds__(kThreads)
gated_rms_kernel(XpGatedRmsArgs a) {
  __shared__ float red[kThreads / 32];
  const float* o = a.o + static_cast<size_t>(blockIdx.x) * a.ld_o;
  const T* gate = reinterpret_cast<const T*>(a.gate) + static_cast<size_t>(blockIdx.x) * a.ld_gate;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<size_t>(blockIdx.x) * a.ld_out;
  float ss = 0.f;
  for (int c = threadIdx.x * N; c < a.cols; c += kThreads * N) {
    float v[N];
    ldv<N>(o + c, v);
#pragma unroll
    for (int j = 0; j < N; ++j) ss += v[j] * v[j];
  }
  const float inv = rsqrtf(block_sum<kThreads>(ss, red) / static_cast<float>(a.cols) + a.eps);
  for (int c = threadIdx.x * N; c < a.cols; c += kThreads * N) {
    float v[N], w[N], g[N];
    ldv<N>(o + c, v);
    ldv<N>(a.weight + c, w);
    ldv<N>(gate + c, g);
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = v[j] * inv * w[j] * sigmoid(g[j]);
    stv<N>(out + c, v);
  }
}

inline bool vec4(const void* p, int64_t ld, int elem_bytes) {
  return p == nullptr || (reinterpret_cast<uintptr_t>(p) % (4 * elem_bytes) == 0 && ld % 4 == 0);
}

template <typename T, int N>
void launch_resid(const XpResidNormArgs& a, cudaStream_t s) {
  if (a.kind == kRms) resid_norm_kernel<T, N, kRms><<<a.rows, kThreads, 0, s>>>(a);
  else if (a.kind == kLayer) resid_norm_kernel<T, N, kLayer><<<a.rows, kThreads, 0, s>>>(a);
  else resid_norm_kernel<T, N, kDynTanh><<<a.rows, kThreads, 0, s>>>(a);
}

inline int done() {
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -100 - static_cast<int>(e);
}

}  // namespace rowops
}  // namespace xpool

using namespace xpool::rowops;

extern "C" int xp_resid_norm(const XpResidNormArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->hidden <= 0 || a->nparts < 0 || a->nparts > 8 || a->kind < 0 || a->kind > 2) return -10;
  if (a->out != nullptr && (a->weight == nullptr || (a->kind == kDynTanh && a->alpha == nullptr))) return -11;
  const int eb = a->f32 ? 4 : 2;
  bool v = a->hidden % 4 == 0 && vec4(a->resid, a->hidden, 4) && vec4(a->gate, a->ld_gate, eb) && vec4(a->table, a->hidden, eb) &&
           vec4(a->weight, 0, 4) && vec4(a->bias, 0, 4) && vec4(a->out, a->ld_out, eb);
  for (int p = 0; p < a->nparts; ++p) v = v && vec4(a->parts[p], a->ld_part, eb);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->f32) v ? launch_resid<float, 4>(*a, s) : launch_resid<float, 1>(*a, s);
  else v ? launch_resid<__nv_bfloat16, 4>(*a, s) : launch_resid<__nv_bfloat16, 1>(*a, s);
  return done();
}

extern "C" int xp_polynorm(const XpPolyNormArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->cols <= 0) return -10;
  const int eb = a->f32 ? 4 : 2;
  const bool v = a->cols % 4 == 0 && vec4(a->z, a->ld_z, eb) && vec4(a->out, a->ld_out, eb);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->f32) {
    if (v) polynorm_kernel<float, 4><<<a->rows, kThreads, 0, s>>>(*a);
    else polynorm_kernel<float, 1><<<a->rows, kThreads, 0, s>>>(*a);
  } else {
    if (v) polynorm_kernel<__nv_bfloat16, 4><<<a->rows, kThreads, 0, s>>>(*a);
    else polynorm_kernel<__nv_bfloat16, 1><<<a->rows, kThreads, 0, s>>>(*a);
  }
  return done();
}

extern "C" int xp_gated_rms(const XpGatedRmsArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->cols <= 0) return -10;
  const int eb = a->f32 ? 4 : 2;
  const bool v = a->cols % 4 == 0 && vec4(a->o, a->ld_o, 4) && vec4(a->weight, 0, 4) && vec4(a->gate, a->ld_gate, eb) &&
                 vec4(a->out, a->ld_out, eb);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->f32) {
    if (v) gated_rms_kernel<float, 4><<<a->rows, kThreads, 0, s>>>(*a);
    else gated_rms_kernel<float, 1><<<a->rows, kThreads, 0, s>>>(*a);
  } else {
    if (v) gated_rms_kernel<__nv_bfloat16, 4><<<a->rows, kThreads, 0, s>>>(*a);
    else gated_rms_kernel<__nv_bfloat16, 1><<<a->rows, kThreads, 0, s>>>(*a);
  }
  return done();
}
