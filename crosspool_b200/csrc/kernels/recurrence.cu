// Linear-attention recurrences whose decays come from the input, with a state per sequence and head (fp32, [dim][vdim], in the
// sequence's slot; a sequence whose first row sits at position 0 starts from zero):
//   gated linear   S = diag(alpha) S + k v^T                                   alpha per key channel
//   delta rule     S = g S;  u = beta (v - S^T k);  S = S + k u^T              g and beta per head
// Decode kernels do a token's whole mixer between its two projections: (convolution, unit vectors, decay map,) state update,
// read-out, norm per head and gate. The state is read once and written once.
// Prefill: sequential kernels here (any sizes, fp32 or bf16); chunked tensor-core kernels in delta_chunked.cu and
// gated_linear_chunked.cu.
#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"
#include "xpool/recurrence.cuh"

namespace xpool {
namespace recur {

using elem::block_sum;
using elem::ld;
using elem::ldv;
using elem::silu;
using elem::st;
using elem::stv;

constexpr int kThreads = 256;

// ------------------------------------------------------------------------------------------ decode
// The state tile of a CTA (one head, one sequence): kThreads threads = column groups of N x row groups; a thread owns rows
// gi, gi + groups, ... of its N columns. PER rows are held in registers (all loads in flight at once); PER = 0 walks the rows
// twice instead, for states too large to hold.
template <int N, int PER>
struct Tile {
  int cols, groups, gi, cj;
  bool on;
  __device__ explicit Tile(int vdim) {
    cols = (vdim + N - 1) / N;
    groups = kThreads / cols > 0 ? kThreads / cols : 1;
    const int step = cols < kThreads ? cols : kThreads;
    gi = threadIdx.x / step;
    cj = threadIdx.x % step;
    on = gi < groups;
  }
};

// rmsnorm(o) * norm * silu(gate) of one head; o in shared memory.
template <typename T>
__device__ __forceinline__ void store_head(const float* o, int vdim, const float* norm, const T* gate, T* out, float eps, float* red) {
  float ss = 0.f;
  for (int c = threadIdx.x; c < vdim; c += kThreads) ss += o[c] * o[c];
  const float inv = rsqrtf(block_sum<kThreads>(ss, red) / static_cast<float>(vdim) + eps);
  for (int c = threadIdx.x; c < vdim; c += kThreads) st(out + c, o[c] * inv * norm[c] * silu(ld(gate + c)));
}

// Column sums over the row groups: part [groups][vdim] -> dst [vdim].
template <typename F>
__device__ __forceinline__ void fold(const float* part, int groups, int vdim, F&& f) {
  for (int c = threadIdx.x; c < vdim; c += kThreads) {
    float t = 0.f;
    for (int i = 0; i < groups; ++i) t += part[i * vdim + c];
    f(c, t);
  }
}

template <typename T, int N, int PER>
__global__ void __launch_bounds__(kThreads)
gated_linear_decode_kernel(XpGatedLinearArgs a) {
  extern __shared__ float sm[];            // q, k, alpha [dim]; a1 [rank]; partial sums [groups][vdim]; o [vdim]
  __shared__ float red[kThreads / 32];
  const int h = blockIdx.x, row = blockIdx.y;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<size_t>(row) * a.ld_out + static_cast<size_t>(h) * a.vdim;
  if (a.slots[row] < 0) {
    for (int c = threadIdx.x; c < a.vdim; c += kThreads) st(out + c, 0.f);
    return;
  }
  const Tile<N, PER> tile(a.vdim);
  float* q_s = sm;
  float* k_s = q_s + a.dim;
  float* al_s = k_s + a.dim;
  float* a1_s = al_s + a.dim;
  float* part = a1_s + (a.rank + 3) / 4 * 4;
  float* o_s = part + tile.groups * a.vdim;
  const bool fresh = a.positions[row] == 0;
  float* S = a.state + (static_cast<size_t>(a.state_slots[row]) * a.heads + h) * a.dim * a.vdim;
  float s[PER > 0 ? PER : 1][N];
  if constexpr (PER > 0) {                 // the state is on its way while the decays are computed
#pragma unroll
    for (int u = 0; u < PER; ++u) {
#pragma unroll
      for (int j = 0; j < N; ++j) s[u][j] = 0.f;
      const int i = tile.gi + u * tile.groups;
      if (tile.on && !fresh && i < a.dim) ldv<N>(S + static_cast<size_t>(i) * a.vdim + tile.cj * N, s[u]);
    }
  }
  const T* proj = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.ld_proj;
  for (int c = threadIdx.x; c < a.rank; c += kThreads) a1_s[c] = ld(proj + a.a_off + c);
  for (int c = threadIdx.x; c < a.dim; c += kThreads) {
    q_s[c] = ld(proj + a.q_off + h * a.dim + c) * a.qscale;
    k_s[c] = ld(proj + a.k_off + h * a.dim + c);
  }
  __syncthreads();
  for (int c = threadIdx.x; c < a.dim; c += kThreads) {
    const T* w = reinterpret_cast<const T*>(a.a2) + static_cast<size_t>(h * a.dim + c) * a.ld_a2;
    float z = a.a2_bias[h * a.dim + c];
    for (int j = 0; j < a.rank; ++j) z = fmaf(ld(w + j), a1_s[j], z);
    al_s[c] = expf(log_decay(z, a.inv_tau));
  }
  __syncthreads();
  const T* v_p = proj + a.v_off + h * a.vdim;
  if (tile.on) {
    for (int cg = tile.cj; cg < tile.cols; cg += kThreads) {
      const int c = cg * N;
      float v[N], acc[N];
      ldv<N>(v_p + c, v);
#pragma unroll
      for (int j = 0; j < N; ++j) acc[j] = 0.f;
      auto update = [&](int i, float (&x)[N]) {
        const float ai = al_s[i], ki = k_s[i], qi = q_s[i];
#pragma unroll
        for (int j = 0; j < N; ++j) {
          x[j] = fmaf(ki, v[j], ai * x[j]);
          acc[j] = fmaf(qi, x[j], acc[j]);
        }
        stv<N>(S + static_cast<size_t>(i) * a.vdim + c, x);
      };
      if constexpr (PER > 0) {
#pragma unroll
        for (int u = 0; u < PER; ++u) {
          const int i = tile.gi + u * tile.groups;
          if (i < a.dim) update(i, s[u]);
        }
      } else {
        for (int i = tile.gi; i < a.dim; i += tile.groups) {
          float x[N];
#pragma unroll
          for (int j = 0; j < N; ++j) x[j] = 0.f;
          if (!fresh) ldv<N>(S + static_cast<size_t>(i) * a.vdim + c, x);
          update(i, x);
        }
      }
#pragma unroll
      for (int j = 0; j < N; ++j) part[tile.gi * a.vdim + c + j] = acc[j];
    }
  }
  __syncthreads();
  fold(part, tile.groups, a.vdim, [&](int c, float t) { o_s[c] = t; });
  store_head<T>(o_s, a.vdim, a.norm, proj + a.g_off + h * a.vdim, out, a.eps, red);
}

// The token at position p reads entries p - 1 .. p - taps + 1 of the ring (mod taps) and writes entry p, which nobody reads in
// this step: heads that share a query and key may all be at work.
template <typename T>
__device__ __forceinline__ float convolved(const XpDeltaArgs& a, const T* x, T* ring, int c, int pos) {
  const float* w = a.conv_w + static_cast<size_t>(c) * a.taps;
  const int channels = 2 * a.kv_heads * a.dim + a.heads * a.vdim;
  float y = w[a.taps - 1] * ld(x);
  for (int j = 1; j < a.taps; ++j)
    if (pos - j >= 0) y = fmaf(w[a.taps - 1 - j], ld(ring + static_cast<size_t>((pos - j) % a.taps) * channels + c), y);
  return silu(y);
}

template <typename T, int N, int PER>
__global__ void __launch_bounds__(kThreads)
delta_decode_kernel(XpDeltaArgs a) {
  extern __shared__ float sm[];            // q, k [dim]; v [vdim]; u [vdim]; partial sums [groups][vdim]
  __shared__ float red[kThreads / 32];
  const int h = blockIdx.x, row = blockIdx.y;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<size_t>(row) * a.ld_out + static_cast<size_t>(h) * a.vdim;
  if (a.slots[row] < 0) {
    for (int c = threadIdx.x; c < a.vdim; c += kThreads) st(out + c, 0.f);
    return;
  }
  const Tile<N, PER> tile(a.vdim);
  float* q_s = sm;
  float* k_s = q_s + a.dim;
  float* v_s = k_s + a.dim;
  float* u_s = v_s + a.vdim;
  float* part = u_s + a.vdim;
  const int pos = a.positions[row];
  const bool fresh = pos == 0;
  const int slot = a.state_slots[row];
  float* S = a.state + (static_cast<size_t>(slot) * a.heads + h) * a.dim * a.vdim;
  float s[PER > 0 ? PER : 1][N];
  if constexpr (PER > 0) {                 // the state is on its way while the convolution runs
#pragma unroll
    for (int u = 0; u < PER; ++u) {
#pragma unroll
      for (int j = 0; j < N; ++j) s[u][j] = 0.f;
      const int i = tile.gi + u * tile.groups;
      if (tile.on && !fresh && i < a.dim) ldv<N>(S + static_cast<size_t>(i) * a.vdim + tile.cj * N, s[u]);
    }
  }
  const T* proj = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.ld_proj;
  const int ratio = a.heads / a.kv_heads, hk = h / ratio, nq = a.kv_heads * a.dim;
  const int channels = 2 * nq + a.heads * a.vdim;
  T* ring = reinterpret_cast<T*>(a.conv_state) + static_cast<size_t>(slot) * a.taps * channels;
  T* mine = ring + static_cast<size_t>(pos % a.taps) * channels;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < 2 * a.dim + a.vdim; i += kThreads) {
    const int which = i < a.dim ? 0 : i < 2 * a.dim ? 1 : 2;
    const int c = which == 0 ? hk * a.dim + i : which == 1 ? nq + hk * a.dim + i - a.dim : 2 * nq + h * a.vdim + i - 2 * a.dim;
    const T* x = proj + (which == 0 ? a.q_off + c : which == 1 ? a.k_off + c - nq : a.v_off + c - 2 * nq);
    const float y = convolved(a, x, ring, c, pos);
    if (which == 2 || h % ratio == 0) mine[c] = *x;
    sm[i] = y;
    if (which == 0) sq += y * y;
    if (which == 1) sk += y * y;
  }
  const float cq = a.qscale * rsqrtf(block_sum<kThreads>(sq, red) + kUnitEps);
  const float ck = rsqrtf(block_sum<kThreads>(sk, red) + kUnitEps);
  for (int i = threadIdx.x; i < a.dim; i += kThreads) q_s[i] *= cq, k_s[i] *= ck;
  const float g = expf(delta_log_decay(ld(proj + a.a_off + h), a.neg_a[h], a.dt_bias[h]));
  const float beta = elem::sigmoid(ld(proj + a.b_off + h));
  __syncthreads();
  // what the decayed state holds under the key
  if (tile.on) {
    for (int cg = tile.cj; cg < tile.cols; cg += kThreads) {
      const int c = cg * N;
      float acc[N];
#pragma unroll
      for (int j = 0; j < N; ++j) acc[j] = 0.f;
      if constexpr (PER > 0) {
#pragma unroll
        for (int u = 0; u < PER; ++u) {
          const int i = tile.gi + u * tile.groups;
          const float ki = i < a.dim ? k_s[i] : 0.f;
#pragma unroll
          for (int j = 0; j < N; ++j) {
            s[u][j] *= g;
            acc[j] = fmaf(ki, s[u][j], acc[j]);
          }
        }
      } else if (!fresh) {
        for (int i = tile.gi; i < a.dim; i += tile.groups) {
          float x[N];
          ldv<N>(S + static_cast<size_t>(i) * a.vdim + c, x);
          const float ki = k_s[i] * g;
#pragma unroll
          for (int j = 0; j < N; ++j) acc[j] = fmaf(ki, x[j], acc[j]);
        }
      }
#pragma unroll
      for (int j = 0; j < N; ++j) part[tile.gi * a.vdim + c + j] = acc[j];
    }
  }
  __syncthreads();
  fold(part, tile.groups, a.vdim, [&](int c, float t) { u_s[c] = beta * (v_s[c] - t); });
  __syncthreads();
  if (tile.on) {
    for (int cg = tile.cj; cg < tile.cols; cg += kThreads) {
      const int c = cg * N;
      float uu[N], acc[N];
#pragma unroll
      for (int j = 0; j < N; ++j) uu[j] = u_s[c + j], acc[j] = 0.f;
      auto update = [&](int i, float (&x)[N]) {
        const float ki = k_s[i], qi = q_s[i];
#pragma unroll
        for (int j = 0; j < N; ++j) {
          x[j] = fmaf(ki, uu[j], x[j]);
          acc[j] = fmaf(qi, x[j], acc[j]);
        }
        stv<N>(S + static_cast<size_t>(i) * a.vdim + c, x);
      };
      if constexpr (PER > 0) {
#pragma unroll
        for (int u = 0; u < PER; ++u) {
          const int i = tile.gi + u * tile.groups;
          if (i < a.dim) update(i, s[u]);
        }
      } else {
        for (int i = tile.gi; i < a.dim; i += tile.groups) {
          float x[N];
#pragma unroll
          for (int j = 0; j < N; ++j) x[j] = 0.f;
          if (!fresh) {
            ldv<N>(S + static_cast<size_t>(i) * a.vdim + c, x);
#pragma unroll
            for (int j = 0; j < N; ++j) x[j] *= g;
          }
          update(i, x);
        }
      }
#pragma unroll
      for (int j = 0; j < N; ++j) part[tile.gi * a.vdim + c + j] = acc[j];
    }
  }
  __syncthreads();
  fold(part, tile.groups, a.vdim, [&](int c, float t) { v_s[c] = t; });
  store_head<T>(v_s, a.vdim, a.norm, proj + a.g_off + h * a.vdim, out, a.eps, red);
}

// ------------------------------------------------------------------------------------------ sequential prefill
// CTA = (32 state columns, head, sequence). Eight lanes share a column's rows (PER each), a warp has four columns, so that a
// token needs no barrier; tokens are staged kBatch at a time.
constexpr int kBatch = 16;

template <typename T, int PER, bool kDelta, typename A>
__global__ void __launch_bounds__(kThreads)
sequential_kernel(A a) {
  extern __shared__ float sm[];            // q, k [kBatch][dim]; alpha [kBatch][dim] (delta: g, beta [kBatch]); v [kBatch][32]
  const int h = blockIdx.y, seq = blockIdx.z;
  const int n = a.q_lens[seq];
  if (n <= 0) return;
  const int r0 = a.q_starts[seq];
  float* q_s = sm;
  float* k_s = q_s + kBatch * a.dim;
  float* al_s = k_s + kBatch * a.dim;
  float* v_s = al_s + (kDelta ? 2 * kBatch : kBatch * a.dim);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rg = lane & 7, col = warp * 4 + (lane >> 3);
  const int c = blockIdx.x * 32 + col;
  const bool on = c < a.vdim;
  float* S = a.state + (static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * a.dim * a.vdim;
  const bool fresh = a.positions[r0] == 0;
  float s[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int d = i * 8 + rg;
    s[i] = on && d < a.dim && !fresh ? S[static_cast<size_t>(d) * a.vdim + c] : 0.f;
  }
  for (int t0 = 0; t0 < n; t0 += kBatch) {
    const int m = min(kBatch, n - t0);
    if constexpr (kDelta) {
      const int hk = h / (a.heads / a.kv_heads), nq = a.kv_heads * a.dim, channels = 2 * nq + a.heads * a.vdim;
      for (int i = threadIdx.x; i < m * a.dim; i += kThreads) {
        const int t = i / a.dim, d = i - t * a.dim, row = r0 + t0 + t;
        const T* p = reinterpret_cast<const T*>(a.qkv) + static_cast<size_t>(row) * channels + hk * a.dim + d;
        const float* f = a.qk_scale + static_cast<size_t>(row) * 2 * a.kv_heads + hk;
        q_s[i] = ld(p) * f[0];
        k_s[i] = ld(p + nq) * f[a.kv_heads];
      }
      for (int i = threadIdx.x; i < m * 32; i += kThreads) {
        const int t = i >> 5, cc = blockIdx.x * 32 + (i & 31);
        v_s[i] = cc < a.vdim ? ld(reinterpret_cast<const T*>(a.qkv) + static_cast<size_t>(r0 + t0 + t) * channels + 2 * nq + h * a.vdim + cc) : 0.f;
      }
      if (threadIdx.x < m) {
        const float* f = a.beta_g + static_cast<size_t>(r0 + t0 + threadIdx.x) * 2 * a.heads + h;
        al_s[threadIdx.x] = expf(f[a.heads]);
        al_s[kBatch + threadIdx.x] = f[0];
      }
    } else {
      for (int i = threadIdx.x; i < m * a.dim; i += kThreads) {
        const int t = i / a.dim, d = i - t * a.dim;
        const size_t row = r0 + t0 + t;
        const T* p = reinterpret_cast<const T*>(a.proj) + row * a.ld_proj + h * a.dim + d;
        q_s[i] = ld(p + a.q_off) * a.qscale;
        k_s[i] = ld(p + a.k_off);
        al_s[i] = expf(log_decay(a.z[row * a.heads * a.dim + h * a.dim + d], a.inv_tau));
      }
      for (int i = threadIdx.x; i < m * 32; i += kThreads) {
        const int t = i >> 5, cc = blockIdx.x * 32 + (i & 31);
        v_s[i] = cc < a.vdim ? ld(reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(r0 + t0 + t) * a.ld_proj + a.v_off + h * a.vdim + cc) : 0.f;
      }
    }
    __syncthreads();
    for (int t = 0; t < m; ++t) {
      float w = v_s[t * 32 + col], o = 0.f;
      const float* kt = k_s + t * a.dim;
      const float* qt = q_s + t * a.dim;
      auto column_sum = [](float x) {
#pragma unroll
        for (int d = 4; d > 0; d >>= 1) x += __shfl_xor_sync(0xffffffffu, x, d);
        return x;
      };
      if constexpr (kDelta) {
        const float g = al_s[t];
        float held = 0.f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
          const int d = i * 8 + rg;
          s[i] *= g;
          if (d < a.dim) held = fmaf(kt[d], s[i], held);
        }
        w = al_s[kBatch + t] * (w - column_sum(held));
      }
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int d = i * 8 + rg;
        if (d < a.dim) {
          s[i] = fmaf(kt[d], w, kDelta ? s[i] : al_s[t * a.dim + d] * s[i]);
          o = fmaf(qt[d], s[i], o);
        }
      }
      o = column_sum(o);
      if (on && rg == 0) reinterpret_cast<float*>(a.out)[static_cast<size_t>(r0 + t0 + t) * a.ld_out + h * a.vdim + c] = o;
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int d = i * 8 + rg;
    if (on && d < a.dim) S[static_cast<size_t>(d) * a.vdim + c] = s[i];
  }
}

// ------------------------------------------------------------------------------------------ delta rule: in front of the recurrence
// CTA = (kPrepRows rows, one head of queries, keys or values, portion): convolution and silu, and for queries and keys the sum
// of squares per row. A thread takes kRun rows of VEC channels, all of its inputs in flight at once. The last CTA column
// computes beta and log g. The CTA of a portion's first rows is the only one that reads the ring (a window reaches back less
// than kPrepRows rows) and puts the portion's last inputs into it when it is done.
constexpr int kPrepRows = 128;
constexpr int kRun = 8;

__device__ __forceinline__ void conv_out(float* p, float y) { *p = silu(y); }
__device__ __forceinline__ void conv_out(__nv_bfloat16* p, float y) { *p = __float2bfloat16_rn(__fdividef(y, 1.f + __expf(-y))); }

// TAPS = 0: any number, inputs read again for every output
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kThreads, 2)
delta_prep_kernel(XpDeltaArgs a) {
  extern __shared__ float sm[];            // sums of squares [kPrepRows][vector columns + 1]
  const int seq = blockIdx.z, n = a.q_lens[seq], t0 = blockIdx.x * kPrepRows;
  if (t0 >= n) return;
  const int rows = min(kPrepRows, n - t0), r0 = a.q_starts[seq] + t0;
  const T* proj = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(r0) * a.ld_proj;
  if (blockIdx.y == 2 * a.kv_heads + a.heads) {
    for (int i = threadIdx.x; i < rows * a.heads; i += kThreads) {
      const int t = i / a.heads, h = i - t * a.heads;
      const T* p = proj + static_cast<size_t>(t) * a.ld_proj + h;
      float* f = a.beta_g + static_cast<size_t>(r0 + t) * 2 * a.heads + h;
      f[0] = elem::sigmoid(ld(p + a.b_off));
      f[a.heads] = delta_log_decay(ld(p + a.a_off), a.neg_a[h], a.dt_bias[h]);
    }
    return;
  }
  const int u = blockIdx.y, nq = a.kv_heads * a.dim, channels = 2 * nq + a.heads * a.vdim;
  const bool is_v = u >= 2 * a.kv_heads;
  const int width = is_v ? a.vdim : a.dim;
  const int ch0 = is_v ? 2 * nq + (u - 2 * a.kv_heads) * a.vdim : u * a.dim;       // first channel (k heads follow q heads)
  const T* x0 = proj + (is_v ? a.v_off + ch0 - 2 * nq : u < a.kv_heads ? a.q_off + ch0 : a.k_off + ch0 - nq);
  const int pos0 = a.positions[r0];
  T* ring = reinterpret_cast<T*>(a.conv_state) + static_cast<size_t>(a.state_slots[seq]) * a.taps * channels;
  T* qkv = reinterpret_cast<T*>(a.qkv) + static_cast<size_t>(r0) * channels + ch0;
  const int vecs = width / VEC, runs = (rows + kRun - 1) / kRun;
  for (int w = threadIdx.x; w < vecs * runs; w += kThreads) {
    const int c = w % vecs * VEC, first = w / vecs * kRun;
    auto input = [&](int t, T (&x)[VEC]) {           // row t of the tile, or what came before it
      const T* p = nullptr;
      if (t0 + t >= 0) p = t < rows ? x0 + static_cast<int64_t>(t) * a.ld_proj : nullptr;
      else if (pos0 + t >= 0) p = ring + static_cast<size_t>((pos0 + t) % a.taps) * channels + ch0;
      if (p != nullptr) {
        ldr<VEC>(p + c, x);
      } else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) st(&x[j], 0.f);
      }
    };
    auto finish = [&](int t, const float (&y)[VEC]) {
      if (t >= rows) return;
      float ss = 0.f;
      T r[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        conv_out(&r[j], y[j]);
        const float f = ld(&r[j]);
        ss += f * f;
      }
      stx<VEC>(qkv + static_cast<size_t>(t) * channels + c, r);
      if (!is_v) sm[t * (vecs + 1) + w % vecs] = ss;
    };
    if constexpr (TAPS > 0) {
      T x[kRun + TAPS - 1][VEC];
      if (t0 + first >= TAPS - 1 && first + kRun <= rows) {      // no branch between the loads
        const T* p = x0 + static_cast<int64_t>(first - (TAPS - 1)) * a.ld_proj + c;
#pragma unroll
        for (int i = 0; i < kRun + TAPS - 1; ++i) ldr<VEC>(p + static_cast<int64_t>(i) * a.ld_proj, x[i]);
      } else {
#pragma unroll
        for (int i = 0; i < kRun + TAPS - 1; ++i) input(first + i - (TAPS - 1), x[i]);
      }
      float wt[VEC][TAPS];
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        if constexpr (TAPS == 4) {
          const float4 f = *reinterpret_cast<const float4*>(a.conv_w + static_cast<size_t>(ch0 + c + j) * 4);
          wt[j][0] = f.x, wt[j][1] = f.y, wt[j][2] = f.z, wt[j][3] = f.w;
        } else {
#pragma unroll
          for (int k = 0; k < TAPS; ++k) wt[j][k] = a.conv_w[static_cast<size_t>(ch0 + c + j) * TAPS + k];
        }
      }
#pragma unroll
      for (int i = 0; i < kRun; ++i) {
        float y[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          y[j] = 0.f;
#pragma unroll
          for (int k = 0; k < TAPS; ++k) y[j] = fmaf(wt[j][k], ld(&x[i + k][j]), y[j]);
        }
        finish(first + i, y);
      }
    } else {
      for (int t = first; t < min(first + kRun, rows); ++t) {
        float y[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) y[j] = 0.f;
        for (int k = 0; k < a.taps; ++k) {
          T x[VEC];
          input(t - k, x);
#pragma unroll
          for (int j = 0; j < VEC; ++j) y[j] = fmaf(a.conv_w[static_cast<size_t>(ch0 + c + j) * a.taps + a.taps - 1 - k], ld(&x[j]), y[j]);
        }
        finish(t, y);
      }
    }
  }
  __syncthreads();
  if (!is_v) {
    const bool is_q = u < a.kv_heads;
    for (int t = threadIdx.x; t < rows; t += kThreads) {
      float ss = 0.f;
      for (int i = 0; i < vecs; ++i) ss += sm[t * (vecs + 1) + i];
      a.qk_scale[static_cast<size_t>(r0 + t) * 2 * a.kv_heads + u] = (is_q ? a.qscale : 1.f) * rsqrtf(ss + kUnitEps);
    }
  }
  if (t0 == 0) {
    const int keep = min(n, a.taps);
    for (int i = threadIdx.x; i < keep * width; i += kThreads) {
      const int j = i / width, c = i - j * width, t = n - 1 - j;
      ring[static_cast<size_t>((pos0 + t) % a.taps) * channels + ch0 + c] = x0[static_cast<size_t>(t) * a.ld_proj + c];
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

inline int row_groups(int vdim, int n) {
  const int cols = (vdim + n - 1) / n;
  return kThreads / cols > 0 ? kThreads / cols : 1;
}

template <typename T, int N, int PER>
int launch(const XpGatedLinearArgs& a, cudaStream_t s) {
  const size_t sm = static_cast<size_t>(3 * a.dim + (a.rank + 3) / 4 * 4 + (row_groups(a.vdim, N) + 1) * a.vdim) * 4;
  const int rc = big_smem(gated_linear_decode_kernel<T, N, PER>, sm);
  if (rc != 0) return rc;
  gated_linear_decode_kernel<T, N, PER><<<dim3(a.heads, a.rows), kThreads, sm, s>>>(a);
  return done();
}
template <typename T, int N, int PER>
int launch(const XpDeltaArgs& a, cudaStream_t s) {
  const size_t sm = static_cast<size_t>(2 * a.dim + (row_groups(a.vdim, N) + 2) * a.vdim) * 4;
  const int rc = big_smem(delta_decode_kernel<T, N, PER>, sm);
  if (rc != 0) return rc;
  delta_decode_kernel<T, N, PER><<<dim3(a.heads, a.rows), kThreads, sm, s>>>(a);
  return done();
}

template <typename T, typename A>
int launch_decode(const A& a, bool vec, cudaStream_t s) {
  const int groups = row_groups(a.vdim, 4), per = (a.dim + groups - 1) / groups;
  if (!vec || a.vdim > 4 * kThreads || per > 32) return vec ? launch<T, 4, 0>(a, s) : launch<T, 1, 0>(a, s);
  if (per <= 4) return launch<T, 4, 4>(a, s);
  if (per <= 8) return launch<T, 4, 8>(a, s);
  if (per <= 16) return launch<T, 4, 16>(a, s);
  return launch<T, 4, 32>(a, s);
}

template <typename T, int PER, bool kDelta, typename A>
int launch_sequential(const A& a, cudaStream_t s) {
  const size_t sm = static_cast<size_t>(kBatch) * ((kDelta ? 2 : 3) * a.dim + (kDelta ? 2 : 0) + 32) * 4;
  const int rc = big_smem(sequential_kernel<T, PER, kDelta, A>, sm);
  if (rc != 0) return rc;
  sequential_kernel<T, PER, kDelta, A><<<dim3((a.vdim + 31) / 32, a.heads, a.seqs), kThreads, sm, s>>>(a);
  return done();
}

template <typename T, bool kDelta, typename A>
int sequential_any(const A& a, cudaStream_t s) {
  if (a.dim <= 64) return launch_sequential<T, 8, kDelta>(a, s);
  if (a.dim <= 128) return launch_sequential<T, 16, kDelta>(a, s);
  if (a.dim <= 256) return launch_sequential<T, 32, kDelta>(a, s);
  if (a.dim <= 512) return launch_sequential<T, 64, kDelta>(a, s);
  return -12;
}

inline bool aligned(const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; }

template <typename T, int VEC, int TAPS>
int launch_prep_taps(const XpDeltaArgs& a, cudaStream_t s) {
  const size_t sm = static_cast<size_t>(kPrepRows) * (a.dim / VEC + 1) * 4;
  const int rc = big_smem(delta_prep_kernel<T, VEC, TAPS>, sm);
  if (rc != 0) return rc;
  delta_prep_kernel<T, VEC, TAPS><<<dim3((a.max_q + kPrepRows - 1) / kPrepRows, 2 * a.kv_heads + a.heads + 1, a.seqs), kThreads, sm, s>>>(a);
  return done();
}

template <typename T, int VEC>
int launch_prep(const XpDeltaArgs& a, cudaStream_t s) {
  if constexpr (VEC > 1) {
    if (a.taps == 4 && aligned(a.conv_w, 16)) return launch_prep_taps<T, VEC, 4>(a, s);
    if (a.taps == 3) return launch_prep_taps<T, VEC, 3>(a, s);
    if (a.taps == 2) return launch_prep_taps<T, VEC, 2>(a, s);
  }
  return launch_prep_taps<T, VEC, 0>(a, s);
}

inline bool delta_ok(const XpDeltaArgs& a) {
  return a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.vdim > 0 && a.taps >= 1 && a.taps <= kPrepRows;
}

}  // namespace recur
}  // namespace xpool

using namespace xpool::recur;

extern "C" int xp_gated_linear_decode(const XpGatedLinearArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->heads <= 0 || a->dim <= 0 || a->vdim <= 0 || a->rank <= 0) return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool v = a->vdim % 4 == 0 && a->ld_proj % 4 == 0 && a->v_off % 4 == 0 && aligned(a->proj, a->f32 ? 16 : 8) && aligned(a->state, 16);
  return a->f32 ? launch_decode<float>(*a, v, s) : launch_decode<__nv_bfloat16>(*a, v, s);
}

extern "C" int xp_delta_decode(const XpDeltaArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (!delta_ok(*a)) return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool v = a->vdim % 4 == 0 && aligned(a->state, 16);
  return a->f32 ? launch_decode<float>(*a, v, s) : launch_decode<__nv_bfloat16>(*a, v, s);
}

extern "C" int xp_delta_prep(const XpDeltaArgs* a, void* stream) {
  if (a->seqs <= 0 || a->max_q <= 0) return 0;
  if (!delta_ok(*a)) return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int vec = a->f32 ? 4 : 8;
  const bool v = a->dim % vec == 0 && a->vdim % vec == 0 && a->ld_proj % vec == 0 && a->q_off % vec == 0 && a->k_off % vec == 0 &&
                 a->v_off % vec == 0 && aligned(a->proj, 16) && aligned(a->qkv, 16) && aligned(a->conv_state, 16);
  if (a->f32) return v ? launch_prep<float, 4>(*a, s) : launch_prep<float, 1>(*a, s);
  return v ? launch_prep<__nv_bfloat16, 8>(*a, s) : launch_prep<__nv_bfloat16, 1>(*a, s);
}

extern "C" int xp_delta_prefill(const XpDeltaArgs* a, void* stream) {
  if (a->seqs <= 0) return 0;
  if (!delta_ok(*a)) return -10;
  if (!a->force_sequential) {
    const int rc = xp_delta_chunked(a, stream);
    if (rc <= 0) return rc;
  }
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->f32 ? sequential_any<float, true>(*a, s) : sequential_any<__nv_bfloat16, true>(*a, s);
}

extern "C" int xp_gated_linear_prefill(const XpGatedLinearArgs* a, void* stream) {
  if (a->seqs <= 0) return 0;
  if (a->heads <= 0 || a->dim <= 0 || a->vdim <= 0) return -10;
  if (!a->force_sequential) {
    const int rc = xp_gated_linear_chunked(a, stream);
    if (rc <= 0) return rc;
  }
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->f32 ? sequential_any<float, false>(*a, s) : sequential_any<__nv_bfloat16, false>(*a, s);
}
