// Decayed linear attention with a recurrent state per sequence and head: S <- decay S + k v^T, o = S^T q, with silu on the
// projected q, k and v. The state is fp32 and lives in the sequence's slot, [dim][vdim] per head; a sequence whose first
// row sits at position 0 starts from zero, so slots are handed out without clearing them.
//   linear_decode      one token per sequence: bound by reading and writing the state once
//   linear_sequential  prefill as a loop over tokens, any sizes, fp32 or bf16 inputs
#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"
#include "xpool/sm100.cuh"

namespace xpool {
namespace linear {

using elem::silu;

constexpr int kThreads = 256;

// ------------------------------------------------------------------------------------------ decode
// CTA = (head, row). N consecutive state columns per thread, rows of the state strided over the thread groups.
template <typename T, int N>
__global__ void __launch_bounds__(kThreads)
linear_decode_kernel(XpLinearAttnArgs a) {
  extern __shared__ float sm[];            // q[dim], k[dim], partial sums [groups][vdim]
  const int h = blockIdx.x, row = blockIdx.y;
  float* out = a.out + static_cast<size_t>(row) * a.heads * a.vdim + static_cast<size_t>(h) * a.vdim;
  if (a.slots[row] < 0) {
    for (int c = threadIdx.x; c < a.vdim; c += kThreads) out[c] = 0.f;
    return;
  }
  float* q_s = sm;
  float* k_s = sm + a.dim;
  float* part = sm + 2 * a.dim;
  const T* proj = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.ld_proj;
  for (int c = threadIdx.x; c < a.dim; c += kThreads) {
    q_s[c] = silu(elem::ld(proj + a.q_off + h * a.dim + c));
    k_s[c] = silu(elem::ld(proj + a.k_off + h * a.dim + c));
  }
  __syncthreads();
  const bool fresh = a.positions[row] == 0;
  const float decay = a.decay[h];
  float* S = a.state + (static_cast<size_t>(a.state_slots[row]) * a.heads + h) * a.dim * a.vdim;
  const int cols = (a.vdim + N - 1) / N;                 // column groups (N divides vdim when N > 1)
  const int groups = kThreads / cols > 0 ? kThreads / cols : 1;
  const int step = cols < kThreads ? cols : kThreads;    // column groups covered at a time
  const int gi = threadIdx.x / step, cj = threadIdx.x % step;
  if (gi < groups) {
    for (int cg = cj; cg < cols; cg += step) {
      const int c = cg * N;
      float v[N], acc[N];
      elem::ldv<N>(proj + a.v_off + h * a.vdim + c, v);
#pragma unroll
      for (int j = 0; j < N; ++j) v[j] = silu(v[j]), acc[j] = 0.f;
#pragma unroll 8
      for (int i = gi; i < a.dim; i += groups) {
        float s[N];
        float* p = S + static_cast<size_t>(i) * a.vdim + c;
        if (fresh) {
#pragma unroll
          for (int j = 0; j < N; ++j) s[j] = 0.f;
        } else {
          elem::ldv<N>(p, s);
        }
        const float ki = k_s[i], qi = q_s[i];
#pragma unroll
        for (int j = 0; j < N; ++j) {
          s[j] = fmaf(ki, v[j], decay * s[j]);
          acc[j] = fmaf(qi, s[j], acc[j]);
        }
        elem::stv<N>(p, s);
      }
#pragma unroll
      for (int j = 0; j < N; ++j) part[gi * a.vdim + c + j] = acc[j];
    }
  }
  __syncthreads();
  for (int c = threadIdx.x; c < a.vdim; c += kThreads) {
    float t = 0.f;
    for (int i = 0; i < groups; ++i) t += part[i * a.vdim + c];
    out[c] = t;
  }
}

// ------------------------------------------------------------------------------------------ sequential prefill
// CTA = (32 state columns, head, sequence): lane = column, the eight warps share the state's rows (PER rows per warp).
constexpr int kBatch = 16;                 // tokens staged at a time

template <typename T, int PER>
__global__ void __launch_bounds__(kThreads)
linear_sequential_kernel(XpLinearAttnArgs a) {
  extern __shared__ float sm[];            // q, k [kBatch][dim]; v [kBatch][32]; partial [kBatch][8][32]
  const int h = blockIdx.y, seq = a.seq0 + blockIdx.z;
  const int n = a.q_lens[seq];
  if (n <= 0) return;
  const int r0 = a.q_starts[seq];
  float* q_s = sm;
  float* k_s = q_s + kBatch * a.dim;
  float* v_s = k_s + kBatch * a.dim;
  float* part = v_s + kBatch * 32;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * 32 + lane;
  const bool on = c < a.vdim;
  const float decay = a.decay[h];
  float* S = a.state + (static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * a.dim * a.vdim;
  const bool fresh = a.positions[r0] == 0;
  float s[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int d = i * 8 + warp;
    s[i] = on && d < a.dim && !fresh ? S[static_cast<size_t>(d) * a.vdim + c] : 0.f;
  }
  for (int t0 = 0; t0 < n; t0 += kBatch) {
    const int m = min(kBatch, n - t0);
    for (int i = threadIdx.x; i < m * a.dim; i += kThreads) {
      const int t = i / a.dim, d = i - t * a.dim;
      const T* p = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(r0 + t0 + t) * a.ld_proj + h * a.dim + d;
      q_s[i] = silu(elem::ld(p + a.q_off));
      k_s[i] = silu(elem::ld(p + a.k_off));
    }
    for (int i = threadIdx.x; i < m * 32; i += kThreads) {
      const int t = i >> 5, cc = blockIdx.x * 32 + (i & 31);
      v_s[i] = cc < a.vdim ? silu(elem::ld(reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(r0 + t0 + t) * a.ld_proj + a.v_off +
                                           h * a.vdim + cc))
                           : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < m; ++t) {
      const float v = v_s[t * 32 + lane];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int d = i * 8 + warp;
        if (d < a.dim) {
          s[i] = fmaf(k_s[t * a.dim + d], v, decay * s[i]);
          o = fmaf(q_s[t * a.dim + d], s[i], o);
        }
      }
      part[(t * 8 + warp) * 32 + lane] = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < m * 32; i += kThreads) {
      const int t = i >> 5, cc = blockIdx.x * 32 + (i & 31);
      if (cc < a.vdim) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) o += part[(t * 8 + w) * 32 + (i & 31)];
        a.out[static_cast<size_t>(r0 + t0 + t) * a.heads * a.vdim + h * a.vdim + cc] = o;
      }
    }
    // the next batch overwrites q, k and v before its first barrier; the partial sums only after it
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int d = i * 8 + warp;
    if (on && d < a.dim) S[static_cast<size_t>(d) * a.vdim + c] = s[i];
  }
}

inline int done() {
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -100 - static_cast<int>(e);
}

template <typename K>
inline int big_smem(K kernel, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  if (bytes > 227 * 1024) return -20;
  return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) == cudaSuccess ? 0 : -21;
}

template <typename T, int N>
int launch_decode(const XpLinearAttnArgs& a, cudaStream_t s) {
  const int cols = (a.vdim + N - 1) / N;
  const int groups = kThreads / cols > 0 ? kThreads / cols : 1;
  const size_t sm = static_cast<size_t>(2 * a.dim + groups * a.vdim) * 4;
  int rc = big_smem(linear_decode_kernel<T, N>, sm);
  if (rc != 0) return rc;
  linear_decode_kernel<T, N><<<dim3(a.heads, a.rows), kThreads, sm, s>>>(a);
  return done();
}

template <typename T, int PER>
int launch_sequential(const XpLinearAttnArgs& a, cudaStream_t s) {
  const size_t sm = static_cast<size_t>(2 * kBatch * a.dim + kBatch * 32 + kBatch * 8 * 32) * 4;
  int rc = big_smem(linear_sequential_kernel<T, PER>, sm);
  if (rc != 0) return rc;
  linear_sequential_kernel<T, PER><<<dim3((a.vdim + 31) / 32, a.heads, a.seqs), kThreads, sm, s>>>(a);
  return done();
}

template <typename T>
int launch_sequential_any(const XpLinearAttnArgs& a, cudaStream_t s) {
  if (a.dim <= 64) return launch_sequential<T, 8>(a, s);
  if (a.dim <= 128) return launch_sequential<T, 16>(a, s);
  if (a.dim <= 256) return launch_sequential<T, 32>(a, s);
  if (a.dim <= 512) return launch_sequential<T, 64>(a, s);
  return -12;
}

}  // namespace linear
}  // namespace xpool

using namespace xpool::linear;

// Rows [0, a->rows), one token each; row r belongs to sequence r (state_slots[r]).
extern "C" int xp_linear_attn_decode(const XpLinearAttnArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->heads <= 0 || a->dim <= 0 || a->vdim <= 0) return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int eb = a->f32 ? 4 : 2;
  const bool v = a->vdim % 4 == 0 && a->ld_proj % 4 == 0 && a->v_off % 4 == 0 && reinterpret_cast<uintptr_t>(a->proj) % (4 * eb) == 0 &&
                 reinterpret_cast<uintptr_t>(a->state) % 16 == 0;
  if (a->f32) return v ? launch_decode<float, 4>(*a, s) : launch_decode<float, 1>(*a, s);
  return v ? launch_decode<__nv_bfloat16, 4>(*a, s) : launch_decode<__nv_bfloat16, 1>(*a, s);
}

// Sequences [seq0, seq0 + seqs) with q_lens[s] rows from q_starts[s].
extern "C" int xp_linear_attn_prefill(const XpLinearAttnArgs* a, void* stream) {
  if (a->seqs <= 0) return 0;
  if (a->heads <= 0 || a->dim <= 0 || a->vdim <= 0) return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->f32 ? launch_sequential_any<float>(*a, s) : launch_sequential_any<__nv_bfloat16>(*a, s);
}
