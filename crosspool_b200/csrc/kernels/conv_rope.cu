// Between the projection and grouped-query attention: a short causal convolution over time on every channel of queries, keys
// and values, rotary positions on the first channels of queries and keys, the padded query layout and the cache rows.
//   conv_rope_decode    one token per sequence, one warp per head
//   conv_rope_prefill   portions: CTA = (kTileRows rows, one head, portion); a thread takes kRun rows of N channels, all of its
//                       inputs in flight at once
// The convolution's inputs are kept per sequence as a ring of `taps` rows, position p in entry p % taps. A decode step reads
// the entries behind its position and writes its own. A portion's first rows are the only ones that reach back into the ring
// (fewer than kTileRows), and the CTA that holds them puts the portion's last inputs into it when it is done.
#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"

namespace xpool {
namespace convrope {

using elem::ld;
using elem::ldv;
using elem::st;
using elem::stv;

constexpr int kThreads = 256;
constexpr int kTileRows = 64;
constexpr int kRun = 8;

// What a block or warp works on: one padded query slot, key head or value head.
struct Unit {
  int n;            // channels (0: padding of a query group)
  int width;        // elements of the destination row
  int in;           // first column in the projection
  int ch;           // first channel of the convolution
  int rotated;      // channels that turn
  int kind;         // 0 query, 1 key, 2 value
  int index;        // query slot or head
};

__device__ __forceinline__ Unit unit_of(const XpConvRopeArgs& a, int u) {
  Unit r;
  const int nq = a.kv_heads * a.group_pad;
  if (u < nq) {
    const int group = a.heads / a.kv_heads, g = u % a.group_pad, h = u / a.group_pad * group + g;
    r.kind = 0, r.index = u;
    r.n = g < group ? a.dim : 0, r.width = a.dq;
    r.ch = h * a.dim, r.in = a.q_off + r.ch, r.rotated = 2 * a.rot_pairs;
  } else {
    const bool is_k = u < nq + a.kv_heads;
    r.index = u - nq - (is_k ? 0 : a.kv_heads);
    r.kind = is_k ? 1 : 2;
    r.n = is_k ? a.dim : a.vdim, r.width = is_k ? a.dq : a.dv;
    r.ch = a.heads * a.dim + (is_k ? 0 : a.kv_heads * a.dim) + r.index * r.n;
    r.in = (is_k ? a.k_off : a.v_off) + r.index * r.n;
    r.rotated = is_k ? 2 * a.rot_pairs : 0;
  }
  return r;
}

__device__ __forceinline__ int channels_of(const XpConvRopeArgs& a) {
  return a.heads * a.dim + (a.own_kv ? a.kv_heads * (a.dim + a.vdim) : 0);
}

// Destination row of a token, or null where the token has no cache row.
template <typename T>
__device__ __forceinline__ T* dest_of(const XpConvRopeArgs& a, const Unit& u, int row) {
  if (u.kind == 0) return reinterpret_cast<T*>(a.q_out) + (static_cast<size_t>(row) * a.kv_heads * a.group_pad + u.index) * a.dq;
  const int slot = a.slots[row];
  if (slot < 0) return nullptr;
  return reinterpret_cast<T*>(u.kind == 1 ? a.k_cache : a.v_cache) + (static_cast<size_t>(slot) * a.kv_heads + u.index) * u.width;
}

// Channel c of a row y after the turn of its position (turn: cos and sin per pair).
__device__ __forceinline__ float turned(const float* y, int c, int pairs, const float2* turn) {
  if (c < pairs) {
    const float2 t = turn[c];
    return y[c] * t.x - y[c + pairs] * t.y;
  }
  const float2 t = turn[c - pairs];
  return y[c] * t.x + y[c - pairs] * t.y;
}

template <typename T, int N>
__global__ void __launch_bounds__(kThreads)
conv_rope_decode_kernel(XpConvRopeArgs a) {
  extern __shared__ float sm[];                      // one row of max(dim, vdim) rounded up per warp
  const int per_row = a.kv_heads * (a.group_pad + (a.own_kv ? 2 : 0));
  const int64_t id = static_cast<int64_t>(blockIdx.x) * (kThreads / 32) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (id >= static_cast<int64_t>(a.rows) * per_row) return;
  const int row = static_cast<int>(id / per_row);
  const Unit u = unit_of(a, static_cast<int>(id % per_row));
  T* dst = dest_of<T>(a, u, row);
  if (dst == nullptr) return;
  float* y_s = sm + (threadIdx.x >> 5) * a.row_floats;
  const int pos = a.positions[row];
  const bool live = a.slots[row] >= 0;               // padding rows own no ring
  const int channels = channels_of(a);
  const T* x = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.ld_proj + u.in;
  T* ring = a.conv_w != nullptr && live ? reinterpret_cast<T*>(a.ring) + static_cast<size_t>(a.state_slots[row]) * a.taps * channels + u.ch : nullptr;
  for (int c = lane * N; c < u.n; c += 32 * N) {
    float y[N], v[N], w[N];
    ldv<N>(x + c, v);
    if (ring != nullptr) {
      stv<N>(ring + static_cast<size_t>(pos % a.taps) * channels + c, v);
      ldv<N>(a.conv_w + static_cast<size_t>(a.taps - 1) * channels + u.ch + c, w);
#pragma unroll
      for (int j = 0; j < N; ++j) y[j] = v[j] * w[j];
      for (int k = 1; k < a.taps && k <= pos; ++k) {
        ldv<N>(ring + static_cast<size_t>((pos - k) % a.taps) * channels + c, v);
        ldv<N>(a.conv_w + static_cast<size_t>(a.taps - 1 - k) * channels + u.ch + c, w);
#pragma unroll
        for (int j = 0; j < N; ++j) y[j] = fmaf(v[j], w[j], y[j]);
      }
    } else {
#pragma unroll
      for (int j = 0; j < N; ++j) y[j] = v[j];
    }
    if (c < u.rotated) stv<N>(y_s + c, y);
    else stv<N>(dst + c, y);
  }
  __syncwarp();
  const float2* turn = reinterpret_cast<const float2*>(a.rot) + static_cast<size_t>(pos < a.rot_positions ? pos : 0) * a.rot_pairs;
  for (int c = lane; c < u.n && c < (u.rotated + N - 1) / N * N; c += 32) st(dst + c, c < u.rotated ? turned(y_s, c, a.rot_pairs, turn) : y_s[c]);
  for (int c = u.n + lane; c < u.width; c += 32) st(dst + c, 0.f);
}

// TAPS = 0: any number, inputs read again for every output
template <typename T, int N, int TAPS>
__global__ void __launch_bounds__(kThreads, 2)
conv_rope_prefill_kernel(XpConvRopeArgs a) {
  extern __shared__ float sm[];                      // [kTileRows][row_floats]
  const int seq = blockIdx.z, n = a.q_lens[seq], t0 = blockIdx.x * kTileRows;
  if (t0 >= n) return;
  const int rows = min(kTileRows, n - t0), r0 = a.q_starts[seq] + t0;
  const Unit u = unit_of(a, blockIdx.y);
  const int channels = channels_of(a), pos0 = a.positions[r0];
  const T* x0 = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(r0) * a.ld_proj + u.in;
  T* ring = a.conv_w != nullptr ? reinterpret_cast<T*>(a.ring) + static_cast<size_t>(a.state_slots[seq]) * a.taps * channels + u.ch : nullptr;
  const int vecs = u.n / N, runs = (rows + kRun - 1) / kRun;
  for (int i = threadIdx.x; i < vecs * runs; i += kThreads) {
    const int c = i % vecs * N, first = i / vecs * kRun;
    auto input = [&](int t, float (&x)[N]) {         // row t of the tile, or what came before it
      const T* p = nullptr;
      if (t0 + t >= 0) p = t < rows ? x0 + static_cast<int64_t>(t) * a.ld_proj : nullptr;
      else if (pos0 + t >= 0) p = ring + static_cast<size_t>((pos0 + t) % a.taps) * channels;
      if (p != nullptr) {
        ldv<N>(p + c, x);
      } else {
#pragma unroll
        for (int j = 0; j < N; ++j) x[j] = 0.f;
      }
    };
    auto finish = [&](int t, const float (&y)[N]) {
      if (t >= rows) return;
      if (c < u.rotated) {
        stv<N>(sm + t * a.row_floats + c, y);
      } else {
        T* dst = dest_of<T>(a, u, r0 + t);
        if (dst != nullptr) stv<N>(dst + c, y);
      }
    };
    if constexpr (TAPS > 0) {
      float x[kRun + TAPS - 1][N], w[TAPS][N];
      if (t0 + first >= TAPS - 1 && first + kRun <= rows) {      // no branch between the loads
        const T* p = x0 + static_cast<int64_t>(first - (TAPS - 1)) * a.ld_proj + c;
#pragma unroll
        for (int k = 0; k < kRun + TAPS - 1; ++k) ldv<N>(p + static_cast<int64_t>(k) * a.ld_proj, x[k]);
      } else {
#pragma unroll
        for (int k = 0; k < kRun + TAPS - 1; ++k) input(first + k - (TAPS - 1), x[k]);
      }
#pragma unroll
      for (int k = 0; k < TAPS; ++k) {
        if (TAPS == 1 && ring == nullptr) {
#pragma unroll
          for (int j = 0; j < N; ++j) w[k][j] = 1.f;
        } else {
          ldv<N>(a.conv_w + static_cast<size_t>(k) * channels + u.ch + c, w[k]);
        }
      }
#pragma unroll
      for (int k = 0; k < kRun; ++k) {
        float y[N];
#pragma unroll
        for (int j = 0; j < N; ++j) {
          y[j] = 0.f;
#pragma unroll
          for (int m = 0; m < TAPS; ++m) y[j] = fmaf(w[m][j], x[k + m][j], y[j]);
        }
        finish(first + k, y);
      }
    } else {
      for (int t = first; t < min(first + kRun, rows); ++t) {
        float y[N], x[N], w[N];
#pragma unroll
        for (int j = 0; j < N; ++j) y[j] = 0.f;
        for (int k = 0; k < a.taps; ++k) {
          input(t - k, x);
          ldv<N>(a.conv_w + static_cast<size_t>(a.taps - 1 - k) * channels + u.ch + c, w);
#pragma unroll
          for (int j = 0; j < N; ++j) y[j] = fmaf(w[j], x[j], y[j]);
        }
        finish(t, y);
      }
    }
  }
  __syncthreads();
  const int rot_vecs = u.n > 0 ? (u.rotated + N - 1) / N : 0;
  for (int i = threadIdx.x; i < rot_vecs * rows; i += kThreads) {
    const int t = i / rot_vecs, c = i % rot_vecs * N, pos = pos0 + t;
    T* dst = dest_of<T>(a, u, r0 + t);
    if (dst == nullptr) continue;
    const float2* turn = reinterpret_cast<const float2*>(a.rot) + static_cast<size_t>(pos < a.rot_positions ? pos : 0) * a.rot_pairs;
    const float* y = sm + t * a.row_floats;
    float v[N];
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = c + j < u.rotated ? turned(y, c + j, a.rot_pairs, turn) : y[c + j];
    stv<N>(dst + c, v);
  }
  const int pad = u.width - u.n;
  for (int i = threadIdx.x; i < pad * rows; i += kThreads) {
    T* dst = dest_of<T>(a, u, r0 + i / pad);
    if (dst != nullptr) st(dst + u.n + i % pad, 0.f);
  }
  if (t0 == 0 && ring != nullptr) {
    const int keep = min(n, a.taps);
    for (int i = threadIdx.x; i < keep * u.n; i += kThreads) {
      const int t = n - 1 - i / u.n, c = i % u.n;
      ring[static_cast<size_t>((pos0 + t) % a.taps) * channels + c] = x0[static_cast<size_t>(t) * a.ld_proj + c];
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

template <typename T, int N>
int launch_decode(const XpConvRopeArgs& a, cudaStream_t s) {
  const int64_t units = static_cast<int64_t>(a.rows) * a.kv_heads * (a.group_pad + (a.own_kv ? 2 : 0));
  const size_t sm = static_cast<size_t>(kThreads / 32) * a.row_floats * 4;
  const int rc = big_smem(conv_rope_decode_kernel<T, N>, sm);
  if (rc != 0) return rc;
  conv_rope_decode_kernel<T, N><<<static_cast<unsigned>((units + kThreads / 32 - 1) / (kThreads / 32)), kThreads, sm, s>>>(a);
  return done();
}

template <typename T, int N, int TAPS>
int launch_taps(const XpConvRopeArgs& a, cudaStream_t s) {
  const size_t sm = static_cast<size_t>(kTileRows) * a.row_floats * 4;
  const int rc = big_smem(conv_rope_prefill_kernel<T, N, TAPS>, sm);
  if (rc != 0) return rc;
  const dim3 grid((a.max_q + kTileRows - 1) / kTileRows, a.kv_heads * (a.group_pad + (a.own_kv ? 2 : 0)), a.seqs);
  conv_rope_prefill_kernel<T, N, TAPS><<<grid, kThreads, sm, s>>>(a);
  return done();
}

template <typename T, int N>
int launch_prefill(const XpConvRopeArgs& a, cudaStream_t s) {
  if (a.conv_w == nullptr || a.taps == 1) return launch_taps<T, N, 1>(a, s);
  if constexpr (N > 1) {
    if (a.taps == 2) return launch_taps<T, N, 2>(a, s);
    if (a.taps == 3) return launch_taps<T, N, 3>(a, s);
    if (a.taps == 4) return launch_taps<T, N, 4>(a, s);
  }
  return launch_taps<T, N, 0>(a, s);
}

inline bool aligned(const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; }

inline int check(XpConvRopeArgs& a) {
  if (a.kv_heads <= 0 || a.heads % a.kv_heads != 0 || a.group_pad < a.heads / a.kv_heads || a.dim <= 0 || a.vdim <= 0 || a.dq < a.dim || a.dv < a.vdim)
    return -10;
  if (a.conv_w != nullptr && (a.taps < 1 || a.taps > kTileRows || a.ring == nullptr)) return -11;
  if (a.rot_pairs < 0 || 2 * a.rot_pairs > a.dim || (a.rot_pairs > 0 && (a.rot == nullptr || a.rot_positions <= 0))) return -12;
  a.row_floats = (2 * a.rot_pairs + 3) / 4 * 4 + 4;  // only what turns is staged
  return 0;
}

inline bool vec4(const XpConvRopeArgs& a) {
  const int eb = a.f32 ? 4 : 2;
  return a.dim % 4 == 0 && a.vdim % 4 == 0 && a.dq % 4 == 0 && a.dv % 4 == 0 && a.ld_proj % 4 == 0 && a.q_off % 4 == 0 && a.k_off % 4 == 0 &&
         a.v_off % 4 == 0 && aligned(a.proj, 4 * eb) && aligned(a.ring, 4 * eb) && aligned(a.q_out, 4 * eb) && aligned(a.k_cache, 4 * eb) &&
         aligned(a.v_cache, 4 * eb) && aligned(a.conv_w, 16);
}

}  // namespace convrope
}  // namespace xpool

using namespace xpool::convrope;

// Rows [0, a->rows), one token each; row r belongs to sequence r (state_slots[r]).
extern "C" int xp_conv_rope_decode(const XpConvRopeArgs* args, void* stream) {
  XpConvRopeArgs a = *args;
  if (a.rows <= 0) return 0;
  const int rc = check(a);
  if (rc != 0) return rc;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool v = vec4(a);
  if (a.f32) return v ? launch_decode<float, 4>(a, s) : launch_decode<float, 1>(a, s);
  return v ? launch_decode<__nv_bfloat16, 4>(a, s) : launch_decode<__nv_bfloat16, 1>(a, s);
}

// Portion s: q_lens[s] rows from row q_starts[s], at most max_q.
extern "C" int xp_conv_rope_prefill(const XpConvRopeArgs* args, void* stream) {
  XpConvRopeArgs a = *args;
  if (a.seqs <= 0 || a.max_q <= 0) return 0;
  const int rc = check(a);
  if (rc != 0) return rc;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool v = vec4(a);
  if (a.f32) return v ? launch_prefill<float, 4>(a, s) : launch_prefill<float, 1>(a, s);
  return v ? launch_prefill<__nv_bfloat16, 4>(a, s) : launch_prefill<__nv_bfloat16, 1>(a, s);
}
