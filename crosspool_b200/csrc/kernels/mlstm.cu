// Matrix memory with exponential gates. Per head, with log gates i = cap tanh(z_i / cap) and f = log sigmoid(cap tanh(z_f / cap)):
//   m' = max(f + m, i)      S' = e^(f + m - m') S + e^(i - m') k v^T      n' = e^(f + m - m') n + e^(i - m') k
//   o  = S'^T q / (max(|n' . q|, e^-m') + 1e-6)
// A head's state [matrix dim x vdim | n dim | m] is fp32 and lives in the sequence's slot; a sequence whose first row sits at
// position 0 starts from zeros.
//   memory_decode      one token per sequence, from the projection to the normed and gated heads
//   memory_gates       prefill, per (head, portion): what the gates of a portion come to (below), and the n and m before it
//   memory_chunked     prefill in chunks of 64 tokens on the tensor cores, bf16 rows
//   memory_sequential  prefill as a loop over tokens, any sizes, fp32 or bf16 rows
//
// Chunks. With F_t the sum of f from the chunk's start to token t, m_0 the maximum before the chunk and
//   a_j = i_j - F_j,   r_t = -max(m_0, a_1 .. a_t)        (so that m_t = F_t - r_t)
// the matrix before the chunk counts with e^(m_0 + r_t) for token t, and token j <= t with e^(a_j + r_t); both are at most 1.
// memory_gates writes a and r (in units of log 2) and m; everything else is parallel over tokens, as in linear_attn.cu.
#include <math_constants.h>

#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"
#include "xpool/mma_sync.cuh"
#include "xpool/recurrence.cuh"
#include "xpool/sm100.cuh"

namespace xpool {
namespace memory {

using elem::block_sum;
using elem::ld;
using elem::ldv;
using elem::sigmoid;
using elem::st;
using elem::stv;

constexpr int kThreads = 256;
constexpr float kFloor = 1e-6f;            // added to what divides the read-out
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float forget_gate(float z, float cap) { return -recur::softplus(-cap * tanhf(z / cap)); }
__device__ __forceinline__ float divisor(float den, float m) { return fmaxf(fabsf(den), expf(-m)) + kFloor; }

// ------------------------------------------------------------------------------------------ decode
// CTA = (head, row). kThreads threads = column groups of N x row groups; a thread owns rows gi, gi + groups, ... of its N
// columns. PER rows are held in registers, all loads in flight at once; PER = 0 goes through the rows one by one.
inline __host__ __device__ int row_groups(int vdim, int n) {
  const int cols = (vdim + n - 1) / n;
  return kThreads / cols > 0 ? kThreads / cols : 1;
}

template <typename T, int N, int PER>
__global__ void __launch_bounds__(kThreads)
memory_decode_kernel(XpMemoryArgs a) {
  extern __shared__ float sm[];            // q, k [dim]; partial sums [groups][vdim]; o [vdim]
  __shared__ float red[kThreads / 32];
  const int h = blockIdx.x, row = blockIdx.y;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<size_t>(row) * a.ld_out + static_cast<size_t>(h) * a.vdim;
  if (a.slots[row] < 0) {
    for (int c = threadIdx.x; c < a.vdim; c += kThreads) st(out + c, 0.f);
    return;
  }
  const int cols = (a.vdim + N - 1) / N, groups = row_groups(a.vdim, N), step = cols < kThreads ? cols : kThreads;
  const int gi = threadIdx.x / step, cj = threadIdx.x % step;
  const bool on = gi < groups;
  float* q_s = sm;
  float* k_s = q_s + (a.dim + 3) / 4 * 4;
  float* part = k_s + (a.dim + 3) / 4 * 4;
  float* o_s = part + groups * a.vdim;
  const bool fresh = a.positions[row] == 0;
  float* S = a.state + (static_cast<size_t>(a.state_slots[row]) * a.heads + h) * a.head_state;
  float* n_p = S + static_cast<size_t>(a.dim) * a.vdim;
  float s[PER > 0 ? PER : 1][N];
  if constexpr (PER > 0) {
#pragma unroll
    for (int u = 0; u < PER; ++u) {
#pragma unroll
      for (int j = 0; j < N; ++j) s[u][j] = 0.f;
      const int i = gi + u * groups;
      if (on && !fresh && i < a.dim) ldv<N>(S + static_cast<size_t>(i) * a.vdim + cj * N, s[u]);
    }
  }
  const T* proj = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.ld_proj;
  const float* z = a.gates + static_cast<size_t>(row) * a.ld_gates + h;
  const float gi_log = input_gate(z[a.i_off], a.cap), gf_log = forget_gate(z[a.f_off], a.cap);
  const float m0 = fresh ? 0.f : n_p[a.dim];
  const float m = fmaxf(gf_log + m0, gi_log);
  const float keep = expf(gf_log + m0 - m), write = expf(gi_log - m);
  float dot = 0.f;
  for (int c = threadIdx.x; c < a.dim; c += kThreads) {
    const float q = ld(proj + a.q_off + h * a.dim + c) * a.qscale, k = ld(proj + a.k_off + h * a.dim + c) * write;
    const float n = fmaf(keep, fresh ? 0.f : n_p[c], k);
    q_s[c] = q, k_s[c] = k;
    n_p[c] = n;
    dot = fmaf(n, q, dot);
  }
  const float inv = 1.f / divisor(block_sum<kThreads>(dot, red), m);   // its barriers stand between reading m and storing it
  if (threadIdx.x == 0) n_p[a.dim] = m;
  const T* v_p = proj + a.v_off + h * a.vdim;
  if (on) {
    for (int cg = cj; cg < cols; cg += kThreads) {
      const int c = cg * N;
      float v[N], acc[N];
      ldv<N>(v_p + c, v);
#pragma unroll
      for (int j = 0; j < N; ++j) acc[j] = 0.f;
      auto update = [&](int i, float (&x)[N]) {
        const float ki = k_s[i], qi = q_s[i];
#pragma unroll
        for (int j = 0; j < N; ++j) {
          x[j] = fmaf(ki, v[j], keep * x[j]);
          acc[j] = fmaf(qi, x[j], acc[j]);
        }
        stv<N>(S + static_cast<size_t>(i) * a.vdim + c, x);
      };
      if constexpr (PER > 0) {
#pragma unroll
        for (int u = 0; u < PER; ++u) {
          const int i = gi + u * groups;
          if (i < a.dim) update(i, s[u]);
        }
      } else {
        for (int i = gi; i < a.dim; i += groups) {
          float x[N];
#pragma unroll
          for (int j = 0; j < N; ++j) x[j] = 0.f;
          if (!fresh) ldv<N>(S + static_cast<size_t>(i) * a.vdim + c, x);
          update(i, x);
        }
      }
#pragma unroll
      for (int j = 0; j < N; ++j) part[gi * a.vdim + c + j] = acc[j];
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < a.vdim; c += kThreads) {
    float t = 0.f;
    for (int i = 0; i < groups; ++i) t += part[i * a.vdim + c];
    t *= inv;
    o_s[c] = t;
    ss += t * t;
  }
  const float rms = rsqrtf(block_sum<kThreads>(ss, red) / static_cast<float>(a.vdim) + a.eps);
  const T* gate = proj + a.g_off + h * a.vdim;
  for (int c = threadIdx.x; c < a.vdim; c += kThreads) st(out + c, o_s[c] * rms * a.norm[h * a.vdim + c] * sigmoid(ld(gate + c)));
}

// ------------------------------------------------------------------------------------------ the gates of a portion
constexpr int kChunk = 64;

__device__ __forceinline__ float* plane(const XpMemoryArgs& a, int which, int h) {
  return a.planes + (static_cast<size_t>(which) * a.heads + h) * a.rows;
}
enum : int { kA = 0, kR = 1, kM = 2 };

// What m becomes over a stretch of tokens: m -> max(m + f, top).
struct Step {
  float f, top;
};
__device__ __forceinline__ Step then(const Step& x, const Step& y) { return {x.f + y.f, fmaxf(x.top + y.f, y.top)}; }

// CTA = (head, portion); a warp takes a chunk at a time, two tokens per lane.
constexpr int kGateThreads = 1024;

__global__ void __launch_bounds__(kGateThreads)
memory_gates_kernel(XpMemoryArgs a) {
  extern __shared__ float sm[];            // per chunk: step (f, top), then the maximum before it
  const int h = blockIdx.x, seq = blockIdx.y, n = a.q_lens[seq];
  if (n <= 0) return;
  const int r0 = a.q_starts[seq], chunks = (n + kChunk - 1) / kChunk;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float2* steps = reinterpret_cast<float2*>(sm);
  const bool fresh = a.positions[r0] == 0;
  const float* n_p = a.state + (static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * a.head_state + static_cast<size_t>(a.dim) * a.vdim;
  float* before = a.before + (static_cast<size_t>(seq) * a.heads + h) * (a.dim + 1);
  for (int c = threadIdx.x; c <= a.dim; c += kGateThreads) before[c] = fresh ? 0.f : n_p[c];
  float* pa = plane(a, kA, h) + r0;
  float* pr = plane(a, kR, h) + r0;
  float* pm = plane(a, kM, h) + r0;
  for (int c = warp; c < chunks; c += kGateThreads / 32) {
    const int t = c * kChunk + lane * 2;
    float i[2], f[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const float* z = a.gates + static_cast<size_t>(r0 + min(t + u, n - 1)) * a.ld_gates + h;
      const bool ok = t + u < n;
      i[u] = ok ? input_gate(z[a.i_off], a.cap) : -CUDART_INF_F;
      f[u] = ok ? forget_gate(z[a.f_off], a.cap) : 0.f;
    }
    float F = f[0] + f[1];
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, F, d);
      if (lane >= d) F += x;
    }
    const float F0 = F - f[1], a0 = i[0] - F0, a1 = i[1] - F;
    float top = fmaxf(a0, a1);
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, top, d);
      if (lane >= d) top = fmaxf(top, x);
    }
    const float prev = __shfl_up_sync(0xffffffffu, top, 1), top0 = lane > 0 ? fmaxf(prev, a0) : a0;
    if (t < n) pa[t] = a0, pr[t] = top0, pm[t] = F0;
    if (t + 1 < n) pa[t + 1] = a1, pr[t + 1] = top, pm[t + 1] = F;
    if (lane == 31) steps[c] = make_float2(F, F + top);
  }
  __syncthreads();
  if (warp == 0) {
    float m = fresh ? 0.f : n_p[a.dim];
    for (int c0 = 0; c0 < chunks; c0 += 32) {
      const int c = c0 + lane;
      Step s{0.f, -CUDART_INF_F};
      if (c < chunks) s = Step{steps[c].x, steps[c].y};
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const Step p{__shfl_up_sync(0xffffffffu, s.f, d), __shfl_up_sync(0xffffffffu, s.top, d)};
        if (lane >= d) s = then(p, s);
      }
      const float after = fmaxf(m + s.f, s.top), at = __shfl_up_sync(0xffffffffu, after, 1);
      if (c < chunks) steps[c].x = lane > 0 ? at : m;
      m = __shfl_sync(0xffffffffu, after, 31);
    }
  }
  __syncthreads();
  for (int t = threadIdx.x; t < n; t += kGateThreads) {
    const float top = fmaxf(steps[t / kChunk].x, pr[t]);
    pa[t] *= kLog2e;
    pr[t] = -top * kLog2e;
    pm[t] += top;
  }
}

// ------------------------------------------------------------------------------------------ sequential prefill
// CTA = (32 state columns, head, portion). Eight lanes share a column's rows (PER each) and carry those rows of n along.
constexpr int kBatch = 16;

template <typename T, int PER>
__global__ void __launch_bounds__(kThreads)
memory_sequential_kernel(XpMemoryArgs a) {
  extern __shared__ float sm[];            // q, k [kBatch][dim]; v [kBatch][32]; keep, write, m [kBatch]
  const int h = blockIdx.y, seq = blockIdx.z;
  const int n = a.q_lens[seq];
  if (n <= 0) return;
  const int r0 = a.q_starts[seq];
  float* q_s = sm;
  float* k_s = q_s + kBatch * a.dim;
  float* v_s = k_s + kBatch * a.dim;
  float* keep_s = v_s + kBatch * 32;
  float* write_s = keep_s + kBatch;
  float* m_s = write_s + kBatch;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rg = lane & 7, col = warp * 4 + (lane >> 3);
  const int c = blockIdx.x * 32 + col;
  const bool lives = c < a.vdim;
  float* S = a.state + (static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * a.head_state;
  const float* before = a.before + (static_cast<size_t>(seq) * a.heads + h) * (a.dim + 1);
  const bool fresh = a.positions[r0] == 0;
  float s[PER], nv[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int d = i * 8 + rg;
    s[i] = lives && d < a.dim && !fresh ? S[static_cast<size_t>(d) * a.vdim + c] : 0.f;
    nv[i] = d < a.dim ? before[d] : 0.f;
  }
  float m = before[a.dim];
  for (int t0 = 0; t0 < n; t0 += kBatch) {
    const int cnt = min(kBatch, n - t0);
    for (int i = threadIdx.x; i < cnt * a.dim; i += kThreads) {
      const int t = i / a.dim, d = i - t * a.dim;
      const T* p = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(r0 + t0 + t) * a.ld_proj + h * a.dim + d;
      q_s[i] = ld(p + a.q_off) * a.qscale;
      k_s[i] = ld(p + a.k_off);
    }
    for (int i = threadIdx.x; i < cnt * 32; i += kThreads) {
      const int t = i >> 5, cc = blockIdx.x * 32 + (i & 31);
      v_s[i] = cc < a.vdim ? ld(reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(r0 + t0 + t) * a.ld_proj + a.v_off + h * a.vdim + cc) : 0.f;
    }
    if (threadIdx.x < 32) {
      float gi = 0.f, gf = 0.f;
      if (lane < cnt) {
        const float* z = a.gates + static_cast<size_t>(r0 + t0 + lane) * a.ld_gates + h;
        gi = input_gate(z[a.i_off], a.cap), gf = forget_gate(z[a.f_off], a.cap);
      }
      for (int t = 0; t < cnt; ++t) {
        const float it = __shfl_sync(0xffffffffu, gi, t), ft = __shfl_sync(0xffffffffu, gf, t);
        const float mn = fmaxf(ft + m, it);
        if (lane == 0) keep_s[t] = expf(ft + m - mn), write_s[t] = expf(it - mn), m_s[t] = mn;
        m = mn;
      }
    }
    __syncthreads();
    for (int t = 0; t < cnt; ++t) {
      const float keep = keep_s[t], write = write_s[t], v = v_s[t * 32 + col];
      float o = 0.f, den = 0.f;
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int d = i * 8 + rg;
        if (d < a.dim) {
          const float k = k_s[t * a.dim + d] * write, q = q_s[t * a.dim + d];
          s[i] = fmaf(k, v, keep * s[i]);
          nv[i] = fmaf(keep, nv[i], k);
          o = fmaf(q, s[i], o);
          den = fmaf(q, nv[i], den);
        }
      }
#pragma unroll
      for (int d = 4; d > 0; d >>= 1) o += __shfl_xor_sync(0xffffffffu, o, d), den += __shfl_xor_sync(0xffffffffu, den, d);
      if (lives && rg == 0) reinterpret_cast<float*>(a.out)[static_cast<size_t>(r0 + t0 + t) * a.ld_out + h * a.vdim + c] = o / divisor(den, m_s[t]);
    }
    __syncthreads();
  }
  float* n_p = S + static_cast<size_t>(a.dim) * a.vdim;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int d = i * 8 + rg;
    if (d >= a.dim) continue;
    if (lives) S[static_cast<size_t>(d) * a.vdim + c] = s[i];
    if (blockIdx.x == 0 && col == 0) n_p[d] = nv[i];
  }
  if (blockIdx.x == 0 && threadIdx.x == 0) n_p[a.dim] = m;
}

// ------------------------------------------------------------------------------------------ chunked prefill
// CTA = (segment of a portion, VS state columns, head, portion); it walks its segment in chunks of 64 tokens with the state in
// registers. Warps: 16 rows of the chunk and half of the output columns; for the state 16-row tiles of it. n is one more
// column of the state: its product with the queries and the sums of the weighted scores give n . q. Weighted scores, weighted
// keys and the state enter their products as bf16 pairs (16 mantissa bits); the sums are fp32. Long portions with few heads are
// cut into segments that run at the same time: what each adds to the state, a scan over them, then the full pass.
using frag::ldsm4;
using frag::ldsm4t;
using frag::mma;
using frag::split2;
using sm100::ex2_approx;

constexpr int kChunkThreads = 256;
constexpr int kGateWords = 3 * kChunk + 4;           // a, r, m of a chunk, and the m before it

template <int D, int VS>
constexpr int chunk_smem_bytes() {
  // q, k [2][64][D + 8]; v [2][64][VS + 8]; state pair [2][D][VS + 8] (column VS is n); gates [2]
  return (4 * kChunk * (D + 8) + 2 * kChunk * (VS + 8) + 2 * D * (VS + 8)) * 2 + 2 * kGateWords * 4;
}

__device__ __forceinline__ void ldsm2t(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}

// kFull: outputs and the state; otherwise only what the segment adds to the state.
template <int D, int VS, bool kFull>
__global__ void __launch_bounds__(kChunkThreads, 1)
memory_chunked_kernel(XpMemoryArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int PD = D + 8, PV = VS + 8;             // pitches: odd multiples of 16 bytes
  constexpr int NO = VS / 16;                        // output tiles of a warp (8 columns each)
  constexpr int MT = D > 128 ? D / 128 : 1;          // state row tiles of a warp
  constexpr int NS = D >= 128 ? VS / 8 : VS / 16;    // state column tiles of a warp
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* k_s = q_s + 2 * kChunk * PD;
  __nv_bfloat16* v_s = k_s + 2 * kChunk * PD;
  __nv_bfloat16* st_s = v_s + 2 * kChunk * PV;       // state: high parts, low parts
  float* gate_s = reinterpret_cast<float*>(st_s + 2 * D * PV);
  const int slices = (a.vdim + VS - 1) / VS;
  const int seg = blockIdx.x / slices, c0 = (blockIdx.x % slices) * VS;
  const int h = blockIdx.y, seq = blockIdx.z;
  const int total = a.q_lens[seq];
  const int first = seg * a.seg_tokens;              // segments are whole chunks long
  if (first >= total) return;
  const bool last = first + a.seg_tokens >= total;
  if (!kFull && last) return;                        // nobody starts behind the last segment
  const int n = min(a.seg_tokens, total - first);
  const int r0 = a.q_starts[seq] + first;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, q4 = lane & 3;
  const int chunks = (n + kChunk - 1) / kChunk;
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(a.proj);
  const float* before = a.before + (static_cast<size_t>(seq) * a.heads + h) * (a.dim + 1);

  // columns behind dim stay zero; nothing below writes them
  if (a.dim < D) {
    const int gap = (D - a.dim) / 8;
    for (int i = threadIdx.x; i < 4 * kChunk * gap; i += kChunkThreads)
      *reinterpret_cast<uint4*>(q_s + (i / gap) * PD + a.dim + (i % gap) * 8) = make_uint4(0, 0, 0, 0);
  }
  auto issue = [&](int c) {
    if (c < chunks) {
      const int b = c & 1, m = min(kChunk, n - c * kChunk);
      const __nv_bfloat16* rows = proj + static_cast<size_t>(r0 + c * kChunk) * a.ld_proj;
      constexpr int kPieces = D / 8, kRows = kChunkThreads / kPieces;       // a row's 16-byte pieces; rows covered at a time
      const int e = (threadIdx.x % kPieces) * 8;
      if (e < a.dim) {
#pragma unroll
        for (int t = threadIdx.x / kPieces; t < kChunk; t += kRows) {
          const bool ok = t < m;
          const __nv_bfloat16* row = rows + static_cast<size_t>(ok ? t : 0) * a.ld_proj + h * a.dim + e;
          if (kFull) frag::copy16(q_s + (b * kChunk + t) * PD + e, row + a.q_off, ok);
          frag::copy16(k_s + (b * kChunk + t) * PD + e, row + a.k_off, ok);
        }
      }
      constexpr int kVPieces = VS / 8, kVRows = kChunkThreads / kVPieces;
      const int ev = (threadIdx.x % kVPieces) * 8;
#pragma unroll
      for (int t = threadIdx.x / kVPieces; t < kChunk; t += kVRows) {
        const bool ok = t < m && c0 + ev < a.vdim;
        frag::copy16(v_s + (b * kChunk + t) * PV + ev, rows + static_cast<size_t>(t < m ? t : 0) * a.ld_proj + a.v_off + h * a.vdim + (ok ? c0 + ev : 0), ok);
      }
      if (threadIdx.x < 3 * kChunk + 1) {            // gates of the chunk, and the m of the token before it
        const int which = threadIdx.x / kChunk, t = threadIdx.x % kChunk, row = r0 + c * kChunk;
        const bool prev = threadIdx.x == 3 * kChunk;
        const float* src = prev ? (first + c * kChunk == 0 ? before + a.dim : plane(a, kM, h) + row - 1) : plane(a, which, h) + row + (t < m ? t : 0);
        const int sz = prev || t < m ? 4 : 0;
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(sm100::smem_u32(gate_s + b * kGateWords + threadIdx.x)), "l"(src), "r"(sz));
      }
    }
    frag::copies_issued();
  };
  issue(0);

  // the warp's part of the state
  const int d0 = D >= 128 ? warp * MT * 16 : (warp & 3) * 16;
  const int s0 = D >= 128 ? 0 : (warp >> 2) * (VS / 2);
  const size_t matrix = static_cast<size_t>(a.dim) * a.vdim;
  float* slot = a.state + (static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * a.head_state;
  float* mid = a.ws + ((static_cast<size_t>(seq) * a.heads + h) * a.segs + seg) * a.head_state;   // used when segs > 1
  const bool zero = !kFull || (a.segs == 1 && a.positions[r0] == 0);
  const float* from = kFull && a.segs > 1 ? mid : slot;
  const float* n_from = a.segs > 1 ? mid + matrix : before;
  float s[MT][NS][4], sn[MT][4];                     // sn: n in column 0 of a tile of its own
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int d = d0 + mt * 16 + g + r * 8, c = c0 + s0 + j * 8 + q4 * 2;
        float2 x = make_float2(0.f, 0.f);
        if (!zero && d < a.dim && c < a.vdim) x = *reinterpret_cast<const float2*>(from + static_cast<size_t>(d) * a.vdim + c);
        s[mt][j][2 * r] = x.x;
        s[mt][j][2 * r + 1] = x.y;
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + mt * 16 + g + r * 8;
      sn[mt][2 * r] = !zero && q4 == 0 && d < a.dim ? n_from[d] : 0.f;
      sn[mt][2 * r + 1] = 0.f;
    }
  }
  auto publish_state = [&]() {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        __nv_bfloat16* row = st_s + (d0 + mt * 16 + g + r * 8) * PV;
        uint32_t hi, lo;
#pragma unroll
        for (int j = 0; j < NS; ++j) {
          split2(s[mt][j][2 * r], s[mt][j][2 * r + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(row + s0 + j * 8 + q4 * 2) = hi;
          *reinterpret_cast<uint32_t*>(row + s0 + j * 8 + q4 * 2 + D * PV) = lo;
        }
        if (s0 == 0) {
          split2(sn[mt][2 * r], sn[mt][2 * r + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(row + VS + q4 * 2) = hi;
          *reinterpret_cast<uint32_t*>(row + VS + q4 * 2 + D * PV) = lo;
        }
      }
  };
  if (kFull) publish_state();

  const int rw = warp & 3, o0 = (warp >> 2) * (VS / 2);   // output rows and columns of the warp
  const uint32_t a_off = frag::a_lane(lane, PD) + rw * 16 * PD * 2;                                     // Q rows of this warp
  const uint32_t b_off = frag::b_lane(lane, PD);                                                        // K as [tokens][dims]
  const uint32_t t_off = frag::bt_lane(lane, PV);                                                       // [k][n] operands, transposed
  const uint32_t n_off = ((lane & 15) * PV + VS) * 2;                                                   // the column of n
  const uint32_t kt_off = frag::at_lane(lane, PD) + d0 * 2;                                             // K^T rows of this warp
  const uint32_t ones = g == 0 ? 0x3f803f80u : 0u;                                                      // B operand: ones in column 0

  for (int c = 0; c < chunks; ++c) {
    const int b = c & 1, m = min(kChunk, n - c * kChunk);
    frag::copies_wait<0>();
    __syncthreads();                                 // chunk c landed, state published, buffers of chunk c - 1 free
    issue(c + 1);
    const float* ga = gate_s + b * kGateWords;       // a, r (log2 units), m
    const float* gr = ga + kChunk;
    const float start = ga[3 * kChunk] * kLog2e;
    const uint32_t kb = sm100::smem_u32(k_s + b * kChunk * PD);
    if constexpr (kFull) {
      const uint32_t qb = sm100::smem_u32(q_s + b * kChunk * PD) + a_off;
      const uint32_t vb = sm100::smem_u32(v_s + b * kChunk * PV) + t_off + o0 * 2;
      const uint32_t sb = sm100::smem_u32(st_s) + t_off + o0 * 2;
      const uint32_t nb = sm100::smem_u32(st_s) + n_off;
      float o[NO][4], p[8][4], dn[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < NO; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) p[j][e] = 0.f;
      // S^T q and n . q, and the scores of this warp's rows against tokens up to its own
#pragma unroll 2
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t qa[4], nh[2], nl[2];
        ldsm4(qb + ks * 32, qa);
        ldsm2t(nb + ks * 16 * PV * 2, nh[0], nh[1]);
        ldsm2t(nb + (D + ks * 16) * PV * 2, nl[0], nl[1]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {                // 16 tokens each
          if (j <= rw) {
            uint32_t kf[4];
            ldsm4(kb + b_off + (j * 16 * PD + ks * 16) * 2, kf);
            mma(p[2 * j], qa, kf[0], kf[1]);
            mma(p[2 * j + 1], qa, kf[2], kf[3]);
          }
        }
        mma(dn, qa, nh[0], nh[1]);
        mma(dn, qa, nl[0], nl[1]);
#pragma unroll
        for (int j = 0; j < NO; j += 2) {
          uint32_t hi[4], lo[4];
          ldsm4t(sb + (ks * 16 * PV + j * 8) * 2, hi);
          ldsm4t(sb + ((D + ks * 16) * PV + j * 8) * 2, lo);
          mma(o[j], qa, hi[0], hi[1]);
          mma(o[j + 1], qa, hi[2], hi[3]);
          mma(o[j], qa, lo[0], lo[1]);
          mma(o[j + 1], qa, lo[2], lo[3]);
        }
      }
      const int i0 = rw * 16 + g;                    // rows i0 and i0 + 8 of the chunk
      const float ri = gr[i0], rj = gr[i0 + 8];
      const float f0 = ex2_approx(start + ri), f1 = ex2_approx(start + rj);
#pragma unroll
      for (int j = 0; j < NO; ++j) o[j][0] *= f0, o[j][1] *= f0, o[j][2] *= f1, o[j][3] *= f1;
      float den0 = 0.f, den1 = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (j <= rw) {
          uint32_t ph[4], pl[4];
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int t = j * 16 + u * 8 + q4 * 2;
            const float2 at = *reinterpret_cast<const float2*>(ga + t);
            auto w = [&](int i, int tok, float e) { return tok <= i ? ex2_approx(e) : 0.f; };
            const float x0 = p[2 * j + u][0] * w(i0, t, at.x + ri), x1 = p[2 * j + u][1] * w(i0, t + 1, at.y + ri);
            const float y0 = p[2 * j + u][2] * w(i0 + 8, t, at.x + rj), y1 = p[2 * j + u][3] * w(i0 + 8, t + 1, at.y + rj);
            den0 += x0 + x1;
            den1 += y0 + y1;
            split2(x0, x1, ph[2 * u], pl[2 * u]);
            split2(y0, y1, ph[2 * u + 1], pl[2 * u + 1]);
          }
#pragma unroll
          for (int v = 0; v < NO; v += 2) {
            uint32_t vf[4];
            ldsm4t(vb + (j * 16 * PV + v * 8) * 2, vf);
            mma(o[v], ph, vf[0], vf[1]);
            mma(o[v + 1], ph, vf[2], vf[3]);
            mma(o[v], pl, vf[0], vf[1]);
            mma(o[v + 1], pl, vf[2], vf[3]);
          }
        }
      }
      if (q4 == 0) den0 = fmaf(f0, dn[0], den0), den1 = fmaf(f1, dn[2], den1);
#pragma unroll
      for (int d = 1; d < 4; d <<= 1) den0 += __shfl_xor_sync(0xffffffffu, den0, d), den1 += __shfl_xor_sync(0xffffffffu, den1, d);
      const float z0 = a.qscale / divisor(den0 * a.qscale, ga[2 * kChunk + i0]), z1 = a.qscale / divisor(den1 * a.qscale, ga[2 * kChunk + i0 + 8]);
#pragma unroll
      for (int v = 0; v < NO; ++v) {
        const int col = c0 + o0 + v * 8 + q4 * 2;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int i = i0 + r * 8;
          if (i < m && col < a.vdim)                 // vdim is even
            *reinterpret_cast<float2*>(reinterpret_cast<float*>(a.out) + static_cast<size_t>(r0 + c * kChunk + i) * a.ld_out + h * a.vdim + col) =
                make_float2(o[v][2 * r] * (r ? z1 : z0), o[v][2 * r + 1] * (r ? z1 : z0));
        }
      }
      if (c + 1 == chunks && !last) break;           // the next segment has its own start state
    }
    if (kFull) __syncthreads();                      // everyone is done with the published state
    const float rn = gr[m - 1], pn = ex2_approx(start + rn);
    const uint32_t vt = sm100::smem_u32(v_s + b * kChunk * PV) + t_off + s0 * 2;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
      for (int j = 0; j < NS; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[mt][j][e] *= pn;
      sn[mt][0] *= pn, sn[mt][2] *= pn;
    }
#pragma unroll
    for (int kk = 0; kk < kChunk / 16; ++kk) {
      // keys of 16 tokens with their weights, as a bf16 pair
      const int t = kk * 16 + q4 * 2;
      auto w = [&](int tok) { return tok < m ? ex2_approx(ga[tok] + rn) : 0.f; };
      const float w0 = w(t), w1 = w(t + 1), w8 = w(t + 8), w9 = w(t + 9);
      uint32_t hi[MT][4], lo[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        uint32_t ka[4];
        ldsm4t(kb + kt_off + (kk * 16 * PD + mt * 16) * 2, ka);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 x = frag::unpack2(ka[i]);
          split2(x.x * (i < 2 ? w0 : w8), x.y * (i < 2 ? w1 : w9), hi[mt][i], lo[mt][i]);
        }
        mma(sn[mt], hi[mt], ones, ones);
        mma(sn[mt], lo[mt], ones, ones);
      }
      constexpr int kGroup = NS < 8 ? NS : 8;        // value tiles whose fragments are live at a time
#pragma unroll
      for (int j0 = 0; j0 < NS; j0 += kGroup) {
        uint32_t vf[kGroup / 2][4];
#pragma unroll
        for (int j = 0; j < kGroup / 2; ++j) ldsm4t(vt + (kk * 16 * PV + (j0 + 2 * j) * 8) * 2, vf[j]);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
          for (int j = 0; j < kGroup; ++j) mma(s[mt][j0 + j], hi[mt], vf[j / 2][(j & 1) * 2], vf[j / 2][(j & 1) * 2 + 1]);
#pragma unroll
          for (int j = 0; j < kGroup; ++j) mma(s[mt][j0 + j], lo[mt], vf[j / 2][(j & 1) * 2], vf[j / 2][(j & 1) * 2 + 1]);
        }
      }
    }
    if (kFull && c + 1 < chunks) publish_state();
  }
  if (kFull && !last) return;
  float* to = kFull ? slot : mid;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + mt * 16 + g + r * 8;
      if (d >= a.dim) continue;
#pragma unroll
      for (int j = 0; j < NS; ++j) {
        const int c = c0 + s0 + j * 8 + q4 * 2;
        if (c < a.vdim) *reinterpret_cast<float2*>(to + static_cast<size_t>(d) * a.vdim + c) = make_float2(s[mt][j][2 * r], s[mt][j][2 * r + 1]);
      }
      if (c0 == 0 && s0 == 0 && q4 == 0) to[matrix + d] = sn[mt][2 * r];
    }
  if (kFull && c0 == 0 && threadIdx.x == 0) slot[matrix + a.dim] = plane(a, kM, h)[r0 + n - 1];
}

// What each segment adds -> the matrix and n before each segment, in place.
__global__ void __launch_bounds__(256)
memory_scan_kernel(XpMemoryArgs a) {
  const int h = blockIdx.y, seq = blockIdx.z;
  const int total = a.q_lens[seq];
  if (total <= 0) return;
  const size_t matrix = static_cast<size_t>(a.dim) * a.vdim;
  const size_t i = blockIdx.x * 256ull + threadIdx.x;
  __shared__ float factor[64];                       // what a whole segment leaves of the state before it
  const int r0 = a.q_starts[seq];
  const float* before = a.before + (static_cast<size_t>(seq) * a.heads + h) * (a.dim + 1);
  const float* pr = plane(a, kR, h) + r0;
  const float* pm = plane(a, kM, h) + r0;
  const int segs = (total + a.seg_tokens - 1) / a.seg_tokens;              // at most 64
  for (int s = threadIdx.x >> 5; s + 1 < segs; s += 8) {                   // the last segment adds to nobody
    float f = 0.f;
    for (int c = threadIdx.x & 31; c < a.seg_tokens / kChunk; c += 32) {
      const int t = s * a.seg_tokens + c * kChunk;
      f += (t == 0 ? before[a.dim] : pm[t - 1]) * kLog2e + pr[t + kChunk - 1];
    }
    f = elem::warp_sum(f);
    if ((threadIdx.x & 31) == 0) factor[s] = ex2_approx(f);
  }
  __syncthreads();
  if (i >= matrix + a.dim) return;
  float* mid = a.ws + (static_cast<size_t>(seq) * a.heads + h) * a.segs * a.head_state + i;
  float x;
  if (i >= matrix) x = before[i - matrix];
  else x = a.positions[r0] == 0 ? 0.f : a.state[(static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * a.head_state + i];
  constexpr int kAhead = 8;                          // loads in flight before the first store
  for (int s0 = 0; s0 < segs; s0 += kAhead) {
    float add[kAhead];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) add[u] = s0 + u + 1 < segs ? mid[static_cast<size_t>(s0 + u) * a.head_state] : 0.f;
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      if (s0 + u >= segs) break;
      mid[static_cast<size_t>(s0 + u) * a.head_state] = x;
      if (s0 + u + 1 < segs) x = fmaf(factor[s0 + u], x, add[u]);
    }
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

template <typename T, int N, int PER>
int launch_decode(const XpMemoryArgs& a, cudaStream_t s) {
  const size_t sm = static_cast<size_t>(2 * ((a.dim + 3) / 4 * 4) + (row_groups(a.vdim, N) + 1) * a.vdim) * 4;
  const int rc = big_smem(memory_decode_kernel<T, N, PER>, sm);
  if (rc != 0) return rc;
  memory_decode_kernel<T, N, PER><<<dim3(a.heads, a.rows), kThreads, sm, s>>>(a);
  return done();
}

template <typename T>
int decode_any(const XpMemoryArgs& a, bool vec, cudaStream_t s) {
  const int groups = row_groups(a.vdim, 4), per = (a.dim + groups - 1) / groups;
  if (!vec || a.vdim > 4 * kThreads || per > 32) return vec ? launch_decode<T, 4, 0>(a, s) : launch_decode<T, 1, 0>(a, s);
  if (per <= 4) return launch_decode<T, 4, 4>(a, s);
  if (per <= 8) return launch_decode<T, 4, 8>(a, s);
  if (per <= 16) return launch_decode<T, 4, 16>(a, s);
  return launch_decode<T, 4, 32>(a, s);
}

template <typename T, int PER>
int launch_sequential(const XpMemoryArgs& a, cudaStream_t s) {
  const size_t sm = static_cast<size_t>(2 * kBatch * a.dim + kBatch * 32 + 3 * kBatch) * 4;
  const int rc = big_smem(memory_sequential_kernel<T, PER>, sm);
  if (rc != 0) return rc;
  memory_sequential_kernel<T, PER><<<dim3((a.vdim + 31) / 32, a.heads, a.seqs), kThreads, sm, s>>>(a);
  return done();
}

template <typename T>
int sequential_any(const XpMemoryArgs& a, cudaStream_t s) {
  if (a.dim <= 64) return launch_sequential<T, 8>(a, s);
  if (a.dim <= 128) return launch_sequential<T, 16>(a, s);
  if (a.dim <= 256) return launch_sequential<T, 32>(a, s);
  if (a.dim <= 512) return launch_sequential<T, 64>(a, s);
  return -12;
}

template <int D, int VS>
int launch_chunked(const XpMemoryArgs& a, cudaStream_t s) {
  constexpr int kSmem = chunk_smem_bytes<D, VS>();
  static_assert(kSmem <= 227 * 1024, "chunk buffers exceed the shared memory of an SM");
  int rc = big_smem(memory_chunked_kernel<D, VS, true>, kSmem);
  if (rc == 0) rc = big_smem(memory_chunked_kernel<D, VS, false>, kSmem);
  if (rc != 0) return rc;
  XpMemoryArgs b = a;
  if (b.segs <= 1) {
    b.segs = 1;
    b.seg_tokens = 0x40000000;
  } else if (b.ws == nullptr || b.segs > 64 || b.seg_tokens <= 0 || b.seg_tokens % kChunk != 0) {
    return -13;
  }
  const dim3 grid((a.vdim + VS - 1) / VS * b.segs, a.heads, a.seqs);
  if (b.segs > 1) {
    memory_chunked_kernel<D, VS, false><<<grid, kChunkThreads, kSmem, s>>>(b);
    memory_scan_kernel<<<dim3((a.dim * a.vdim + a.dim + 255) / 256, a.heads, a.seqs), 256, 0, s>>>(b);
  }
  memory_chunked_kernel<D, VS, true><<<grid, kChunkThreads, kSmem, s>>>(b);
  return done();
}

template <int D>
int launch_chunked_any(const XpMemoryArgs& a, cudaStream_t s) {
  if (a.vdim <= 32) return launch_chunked<D, 32>(a, s);
  if (a.vdim <= 64) return launch_chunked<D, 64>(a, s);
  return launch_chunked<D, 128>(a, s);
}

inline bool aligned(const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; }
inline bool sizes_ok(const XpMemoryArgs& a) {
  return a.heads > 0 && a.dim > 0 && a.vdim > 0 && a.cap > 0.f && a.head_state >= a.dim * a.vdim + a.dim + 1 && a.gates != nullptr;
}

}  // namespace memory
}  // namespace xpool

using namespace xpool::memory;

// Rows [0, a->rows), one token each; row r belongs to sequence r (state_slots[r]).
extern "C" int xp_memory_decode(const XpMemoryArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (!sizes_ok(*a) || a->norm == nullptr) return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool v = a->vdim % 4 == 0 && a->ld_proj % 4 == 0 && a->v_off % 4 == 0 && a->head_state % 4 == 0 && aligned(a->proj, a->f32 ? 16 : 8) &&
                 aligned(a->state, 16);
  return a->f32 ? decode_any<float>(*a, v, s) : decode_any<__nv_bfloat16>(*a, v, s);
}

// Portion s: q_lens[s] rows from row q_starts[s], at most max_q. segs > 1: every portion has at most segs * seg_tokens rows.
extern "C" int xp_memory_prefill(const XpMemoryArgs* a, void* stream) {
  if (a->seqs <= 0 || a->max_q <= 0) return 0;
  if (!sizes_ok(*a) || a->planes == nullptr || a->before == nullptr) return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const size_t sm = static_cast<size_t>((a->max_q + kChunk - 1) / kChunk) * 8;
  int rc = big_smem(memory_gates_kernel, sm);
  if (rc != 0) return rc;
  memory_gates_kernel<<<dim3(a->heads, a->seqs), kGateThreads, sm, s>>>(*a);
  if (a->f32) return sequential_any<float>(*a, s);
  const bool chunked = !a->force_sequential && a->dim <= 256 && a->dim % 8 == 0 && a->vdim % 8 == 0 && a->ld_proj % 8 == 0 && a->q_off % 8 == 0 &&
                       a->k_off % 8 == 0 && a->v_off % 8 == 0 && a->ld_out % 2 == 0 && a->head_state % 2 == 0 && aligned(a->proj, 16) &&
                       aligned(a->out, 8) && aligned(a->state, 8);
  if (!chunked) return sequential_any<__nv_bfloat16>(*a, s);
  if (a->dim <= 64) return launch_chunked_any<64>(*a, s);
  if (a->dim <= 128) return launch_chunked_any<128>(*a, s);
  return launch_chunked<256, 32>(*a, s);
}
