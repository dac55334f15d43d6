// Row-wise kernels of layered decoders, one CTA per token row, everything computed in fp32:
//   resid_norm   [embedding gather | residual += sublayer output * sigmoid(gate)] -> norm -> activation row
//   polynorm     a N(z) + b N(z^2) + c N(z^3) + e, N dividing the row by its root mean square
//   gated_rms    rmsnorm(o) * w * sigmoid(gate)
//   post_norm    residual += rmsnorm(sublayer output, or the mean of normed branches) * w [-> norm] -> activation row
//   head_gate    rmsnorm per head * w * silu(gate) or sigmoid(gate), one warp per head
//   glu_f32      gated activation of fp32 models (bf16 has it in the product's epilogue)
//   gate_mul     activation times another row, row times sigmoid, squared relu; fp32 models (bf16: the product's epilogue)
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

// A row's elements per thread, kept in registers between the reductions.
constexpr int kPost = 16;

template <typename T, int N, int THREADS>
__global__ void __launch_bounds__(THREADS)
post_norm_kernel(XpPostNormArgs a) {
  __shared__ float red[THREADS / 32];
  const int i = blockIdx.x;
  const int r = a.sel != nullptr ? a.sel[i] : i;
  float* resid = a.resid + static_cast<size_t>(r) * a.hidden;
  const float n = static_cast<float>(a.hidden);
  float y[kPost / N][N], z[kPost / N][N];
  auto each = [&](auto&& f) {
#pragma unroll
    for (int it = 0; it < kPost / N; ++it) {
      const int c = (it * THREADS + threadIdx.x) * N;
      if (c < a.hidden) f(it, c);
    }
  };
  if (a.ids != nullptr) {
    int id = a.ids[r];
    if (id < 0 || id >= a.vocab) id = 0;
    const T* row = reinterpret_cast<const T*>(a.table) + static_cast<size_t>(id) * a.hidden;
    const float es = a.embed_scale == 0.f ? 1.f : a.embed_scale;
    each([&](int it, int c) {
      ldv<N>(row + c, y[it]);
#pragma unroll
      for (int j = 0; j < N; ++j) y[it][j] *= es;
    });
  } else {
    const T* b0 = reinterpret_cast<const T*>(a.branches[0]) + static_cast<size_t>(r) * a.ld_branch[0];
    float s0 = 0.f, s1 = 0.f;
    each([&](int it, int c) {
      ldv<N>(b0 + c, y[it]);
#pragma unroll
      for (int j = 0; j < N; ++j) s0 += y[it][j] * y[it][j];
    });
    if (a.branch_w[0] != nullptr) {
      const bool two = a.nbranches == 2;
      const T* b1 = reinterpret_cast<const T*>(a.branches[1]) + static_cast<size_t>(r) * a.ld_branch[1];
      if (two) {
        each([&](int it, int c) {
          ldv<N>(b1 + c, z[it]);
#pragma unroll
          for (int j = 0; j < N; ++j) s1 += z[it][j] * z[it][j];
        });
      }
      const float share = two ? 0.5f : 1.f;
      const float i0 = share * rsqrtf(block_sum<THREADS>(s0, red) / n + a.eps);
      const float i1 = two ? share * rsqrtf(block_sum<THREADS>(s1, red) / n + a.eps) : 0.f;
      s0 = 0.f;
      each([&](int it, int c) {
        float w[N];
        ldv<N>(a.branch_w[0] + c, w);
#pragma unroll
        for (int j = 0; j < N; ++j) y[it][j] *= i0 * w[j];
        if (two) {
          ldv<N>(a.branch_w[1] + c, w);
#pragma unroll
          for (int j = 0; j < N; ++j) y[it][j] = fmaf(z[it][j] * i1, w[j], y[it][j]);
        }
#pragma unroll
        for (int j = 0; j < N; ++j) s0 += y[it][j] * y[it][j];
      });
    }
    const float inv = rsqrtf(block_sum<THREADS>(s0, red) / n + a.eps);
    each([&](int it, int c) {
      float w[N], v[N];
      ldv<N>(a.weight + c, w);
      ldv<N>(resid + c, v);
#pragma unroll
      for (int j = 0; j < N; ++j) y[it][j] = fmaf(y[it][j] * inv, w[j], v[j]);
    });
  }
  if (a.sel == nullptr) each([&](int it, int c) { stv<N>(resid + c, y[it]); });
  if (a.out == nullptr) return;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<size_t>(i) * a.ld_out;
  if (a.out_weight != nullptr) {
    float s = 0.f;
    each([&](int it, int c) {
#pragma unroll
      for (int j = 0; j < N; ++j) s += y[it][j] * y[it][j];
    });
    const float inv = rsqrtf(block_sum<THREADS>(s, red) / n + a.eps);
    each([&](int it, int c) {
      float w[N];
      ldv<N>(a.out_weight + c, w);
#pragma unroll
      for (int j = 0; j < N; ++j) y[it][j] *= inv * w[j];
    });
  }
  each([&](int it, int c) { stv<N>(out + c, y[it]); });
}

template <typename T, int N>
__global__ void __launch_bounds__(kThreads)
head_gate_kernel(XpHeadGateArgs a) {
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * (kThreads / 32) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= static_cast<int64_t>(a.rows) * a.heads) return;
  const int row = static_cast<int>(unit / a.heads), h = static_cast<int>(unit % a.heads);
  const float* o = a.o + static_cast<size_t>(row) * a.ld_o + h * a.dim;
  const T* gate = reinterpret_cast<const T*>(a.gate) + static_cast<size_t>(row) * a.ld_gate + h * a.dim;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<size_t>(row) * a.ld_out + h * a.dim;
  const float* weight = a.weight + (a.per_head_weight ? h * a.dim : 0);
  float ss = 0.f;
  for (int c = lane * N; c < a.dim; c += 32 * N) {
    float v[N];
    ldv<N>(o + c, v);
#pragma unroll
    for (int j = 0; j < N; ++j) ss += v[j] * v[j];
  }
  const float inv = rsqrtf(elem::warp_sum(ss) / static_cast<float>(a.dim) + a.eps);
  for (int c = lane * N; c < a.dim; c += 32 * N) {
    float v[N], w[N], g[N];
    ldv<N>(o + c, v);
    ldv<N>(weight + c, w);
    ldv<N>(gate + c, g);
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = v[j] * inv * w[j] * (a.sigmoid_gate ? sigmoid(g[j]) : elem::silu(g[j]));
    stv<N>(out + c, v);
  }
}

__device__ __forceinline__ float gated(float g, float alpha, float cubic) { return g / (1.f + expf(-alpha * g * fmaf(cubic * g, g, 1.f))); }

__global__ void __launch_bounds__(kThreads)
glu_f32_kernel(XpGluArgs a) {
  const int c = blockIdx.x * kThreads + threadIdx.x;
  if (c >= a.cols) return;
  for (int r = blockIdx.y; r < a.rows; r += gridDim.y) {
    const float* z = a.z + static_cast<size_t>(r) * a.ld_z;
    const float lim = a.limit > 0.f ? a.limit : 3.0e38f;
    const float g = fminf(z[c], lim), u = fminf(fmaxf(z[a.cols + c], -lim), lim);
    a.out[static_cast<size_t>(r) * a.ld_out + c] = gated(g, a.alpha, a.cubic) * (u + a.up_add);
  }
}

__global__ void __launch_bounds__(kThreads)
gate_mul_f32_kernel(XpGateMulArgs a) {
  const int c = blockIdx.x * kThreads + threadIdx.x;
  if (c >= a.cols) return;
  for (int r = blockIdx.y; r < a.rows; r += gridDim.y) {
    const float z = a.z[static_cast<size_t>(r) * a.ld_z + c], e = a.kind == 2 ? 0.f : a.e[static_cast<size_t>(r) * a.ld_e + c];
    a.out[static_cast<size_t>(r) * a.ld_out + c] = a.kind == 2 ? fmaxf(z, 0.f) * fmaxf(z, 0.f) : a.kind == 1 ? z * sigmoid(e) : gated(z, a.alpha, a.cubic) * e;
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

template <typename T, int N>
int launch_post(const XpPostNormArgs& a, cudaStream_t s) {
  if (a.hidden <= 256 * kPost) post_norm_kernel<T, N, 256><<<a.rows, 256, 0, s>>>(a);
  else if (a.hidden <= 512 * kPost) post_norm_kernel<T, N, 512><<<a.rows, 512, 0, s>>>(a);
  else if (a.hidden <= 1024 * kPost) post_norm_kernel<T, N, 1024><<<a.rows, 1024, 0, s>>>(a);
  else return -12;
  return 0;
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

extern "C" int xp_post_norm(const XpPostNormArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->hidden <= 0 || (a->ids == nullptr && (a->nbranches < 1 || a->nbranches > 2 || a->weight == nullptr))) return -10;
  if (a->nbranches == 2 && (a->branch_w[0] == nullptr || a->branch_w[1] == nullptr)) return -11;
  const int eb = a->f32 ? 4 : 2;
  bool v = a->hidden % 4 == 0 && vec4(a->resid, a->hidden, 4) && vec4(a->table, a->hidden, eb) && vec4(a->weight, 0, 4) &&
           vec4(a->out_weight, 0, 4) && vec4(a->out, a->ld_out, eb);
  for (int i = 0; i < a->nbranches; ++i) v = v && vec4(a->branches[i], a->ld_branch[i], eb) && vec4(a->branch_w[i], 0, 4);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  int rc;
  if (a->f32) rc = v ? launch_post<float, 4>(*a, s) : launch_post<float, 1>(*a, s);
  else rc = v ? launch_post<__nv_bfloat16, 4>(*a, s) : launch_post<__nv_bfloat16, 1>(*a, s);
  return rc != 0 ? rc : done();
}

extern "C" int xp_head_gate(const XpHeadGateArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->heads <= 0 || a->dim <= 0) return -10;
  const int eb = a->f32 ? 4 : 2;
  const bool v = a->dim % 4 == 0 && vec4(a->o, a->ld_o, 4) && vec4(a->weight, 0, 4) && vec4(a->gate, a->ld_gate, eb) &&
                 vec4(a->out, a->ld_out, eb);
  const int64_t units = static_cast<int64_t>(a->rows) * a->heads;
  const unsigned grid = static_cast<unsigned>((units + kThreads / 32 - 1) / (kThreads / 32));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->f32) {
    if (v) head_gate_kernel<float, 4><<<grid, kThreads, 0, s>>>(*a);
    else head_gate_kernel<float, 1><<<grid, kThreads, 0, s>>>(*a);
  } else {
    if (v) head_gate_kernel<__nv_bfloat16, 4><<<grid, kThreads, 0, s>>>(*a);
    else head_gate_kernel<__nv_bfloat16, 1><<<grid, kThreads, 0, s>>>(*a);
  }
  return done();
}

extern "C" int xp_glu_f32(const XpGluArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->cols <= 0) return -10;
  const dim3 grid((a->cols + kThreads - 1) / kThreads, a->rows < 65535 ? a->rows : 65535);
  glu_f32_kernel<<<grid, kThreads, 0, reinterpret_cast<cudaStream_t>(stream)>>>(*a);
  return done();
}

extern "C" int xp_gate_mul_f32(const XpGateMulArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->cols <= 0 || a->kind < 0 || a->kind > 2 || (a->kind != 2 && a->e == nullptr)) return -10;
  const dim3 grid((a->cols + kThreads - 1) / kThreads, a->rows < 65535 ? a->rows : 65535);
  gate_mul_f32_kernel<<<grid, kThreads, 0, reinterpret_cast<cudaStream_t>(stream)>>>(*a);
  return done();
}
