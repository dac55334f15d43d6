// Grouped-query attention: the row kernel of the form without positions between the projection and the attention kernels, and the plain
// attention kernel for sizes and types that the tensor-core kernels (attn_decode.cu, attn_prefill_umma.cu) do not cover.
#include <math_constants.h>

#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"

namespace xpool {
namespace grouped {

using elem::ld;
using elem::st;

constexpr int kPrepThreads = 256;
constexpr int kAttnWarps = 4;

// One warp per head slot of a row: padded query heads, then keys, then values.
template <typename T>
__global__ void __launch_bounds__(kPrepThreads)
grouped_prep_kernel(XpGroupedPrepArgs a) {
  const int per_row = a.kv_heads * (a.group_pad + 2);
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * (kPrepThreads / 32) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= static_cast<int64_t>(a.rows) * per_row) return;
  const int row = static_cast<int>(unit / per_row), u = static_cast<int>(unit % per_row);
  const int nq = a.kv_heads * a.group_pad;
  const T* proj = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.ld_proj;
  const T* src = nullptr;
  T* dst;
  const float* norm = nullptr;
  int n, width;
  if (u < nq) {
    const int group = a.heads / a.kv_heads, g = u % a.group_pad;
    if (g < group) src = proj + a.q_off + (u / a.group_pad * group + g) * a.dim;
    dst = reinterpret_cast<T*>(a.q_out) + (static_cast<size_t>(row) * nq + u) * a.dq;
    norm = a.q_norm, n = a.dim, width = a.dq;
  } else {
    const int slot = a.slots[row];
    if (slot < 0) return;
    const bool is_k = u < nq + a.kv_heads;
    const int h = u - nq - (is_k ? 0 : a.kv_heads);
    n = is_k ? a.dim : a.vdim;
    width = is_k ? a.dq : a.dv;
    src = proj + (is_k ? a.k_off : a.v_off) + h * n;
    dst = reinterpret_cast<T*>(is_k ? a.k_cache : a.v_cache) + (static_cast<size_t>(slot) * a.kv_heads + h) * width;
    if (is_k) norm = a.k_norm;
  }
  float inv = 1.f;
  if (src != nullptr && norm != nullptr) {
    float ss = 0.f;
    for (int c = lane; c < n; c += 32) {
      const float x = ld(src + c);
      ss += x * x;
    }
    inv = rsqrtf(elem::warp_sum(ss) / static_cast<float>(n) + a.eps);
  }
  for (int c = lane; c < width; c += 32) {
    float x = 0.f;
    if (src != nullptr && c < n) {
      x = ld(src + c);
      if (norm != nullptr) x *= inv * norm[c];
    }
    st(dst + c, x);
  }
}

// CTA = (query head, row). A warp takes 32 tokens at a time: lane = token for the scores, lane = value column for the sums.
template <typename T>
__global__ void __launch_bounds__(kAttnWarps * 32)
grouped_attn_kernel(XpGroupedAttnArgs a) {
  extern __shared__ float sm[];            // query [dim]; per warp: accumulators [vdim], maximum, sum
  const int h = blockIdx.x, row = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<size_t>(row) * a.ld_out + h * a.vdim;
  if (a.slots[row] < 0) {
    for (int c = threadIdx.x; c < a.vdim; c += kAttnWarps * 32) st(out + c, 0.f);
    return;
  }
  const int group = a.heads / a.kv_heads, hk = h / group;
  const T* q = reinterpret_cast<const T*>(a.q) + ((static_cast<size_t>(row) * a.kv_heads + hk) * a.group_pad + h % group) * a.dq;
  float* q_s = sm;
  float* acc_s = sm + a.dim + warp * (a.vdim + 2);
  for (int c = threadIdx.x; c < a.dim; c += kAttnWarps * 32) q_s[c] = ld(q + c) * a.scale;
  for (int c = lane; c < a.vdim; c += 32) acc_s[c] = 0.f;
  __syncthreads();
  const int* table = a.block_table + static_cast<size_t>(a.row_seq != nullptr ? a.row_seq[row] : row) * a.max_blocks;
  const int len = a.positions[row] + 1;
  const T* kc = reinterpret_cast<const T*>(a.k_cache);
  const T* vc = reinterpret_cast<const T*>(a.v_cache);
  // the kept first tokens in whole steps of 32, then the step in which the window begins and those behind it
  const int lo = a.window > 0 && len > a.window ? len - a.window : 0;
  const int head = min((a.keep_first + 31) / 32, lo / 32) * 32, skip = lo / 32 * 32 - head;
  float m = -CUDART_INF_F, l = 0.f;
  for (int v0 = warp * 32; v0 + (v0 < head ? 0 : skip) < len; v0 += kAttnWarps * 32) {
    const int t0 = v0 + (v0 < head ? 0 : skip), t = t0 + lane;
    const bool on = t < len && (t >= lo || t < a.keep_first);
    const int tt = t < len ? t : t0;
    const size_t tok = (static_cast<size_t>(table[tt / a.page_size]) * a.page_size + tt % a.page_size) * a.kv_heads + hk;
    const T* k = kc + tok * a.dq;
    float s = 0.f;
    for (int c = 0; c < a.dim; ++c) s = fmaf(q_s[c], ld(k + c), s);
    if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
    if (!on) s = -CUDART_INF_F;
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float mn = fmaxf(m, mx), corr = m == -CUDART_INF_F ? 0.f : expf(m - mn);
    const float p = on ? expf(s - mn) : 0.f;
    l = l * corr + elem::warp_sum(p);
    m = mn;
    const int live = min(32, len - t0);
    for (int c = lane; c - lane < a.vdim; c += 32) {       // every lane takes part in the shuffles
      float v = c < a.vdim ? acc_s[c] * corr : 0.f;
      for (int j = 0; j < live; ++j) {
        const float pj = __shfl_sync(0xffffffffu, p, j);
        const size_t tj = __shfl_sync(0xffffffffu, static_cast<unsigned long long>(tok), j);
        if (c < a.vdim) v = fmaf(pj, ld(vc + tj * a.dv + c), v);
      }
      if (c < a.vdim) acc_s[c] = v;
    }
  }
  if (lane == 0) acc_s[a.vdim] = m, acc_s[a.vdim + 1] = l;
  __syncthreads();
  const float* all = sm + a.dim;
  const int step = a.vdim + 2;
  float mm = -CUDART_INF_F, ll = 0.f;
  for (int w = 0; w < kAttnWarps; ++w) mm = fmaxf(mm, all[w * step + a.vdim]);
  for (int w = 0; w < kAttnWarps; ++w) {
    const float mw = all[w * step + a.vdim];
    if (mw != -CUDART_INF_F) ll += all[w * step + a.vdim + 1] * expf(mw - mm);
  }
  float f = 1.f / ll;
  const T* gate = a.gate != nullptr ? reinterpret_cast<const T*>(a.gate) + static_cast<size_t>(row) * a.ld_gate : nullptr;
  if (gate != nullptr && !a.gate_elems) f *= elem::sigmoid(ld(gate + h));
  for (int c = threadIdx.x; c < a.vdim; c += kAttnWarps * 32) {
    float v = 0.f;
    for (int w = 0; w < kAttnWarps; ++w) {
      const float mw = all[w * step + a.vdim];
      if (mw != -CUDART_INF_F) v += all[w * step + c] * expf(mw - mm);
    }
    if (gate != nullptr && a.gate_elems) v *= elem::sigmoid(ld(gate + h * a.vdim + c));
    st(out + c, v * f);
  }
}

inline int done() {
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -100 - static_cast<int>(e);
}

}  // namespace grouped
}  // namespace xpool

using namespace xpool::grouped;

extern "C" int xp_grouped_prep(const XpGroupedPrepArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->group_pad < a->heads / a->kv_heads || a->dq < a->dim || a->dv < a->vdim) return -10;
  const int64_t units = static_cast<int64_t>(a->rows) * a->kv_heads * (a->group_pad + 2);
  const unsigned grid = static_cast<unsigned>((units + kPrepThreads / 32 - 1) / (kPrepThreads / 32));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->f32) grouped_prep_kernel<float><<<grid, kPrepThreads, 0, s>>>(*a);
  else grouped_prep_kernel<__nv_bfloat16><<<grid, kPrepThreads, 0, s>>>(*a);
  return done();
}

extern "C" int xp_grouped_attn(const XpGroupedAttnArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->rows > 65535) return -10;
  const size_t smem = static_cast<size_t>(a->dim + kAttnWarps * (a->vdim + 2)) * 4;
  if (smem > 48 * 1024) return -11;
  const dim3 grid(a->heads, a->rows);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->f32) grouped_attn_kernel<float><<<grid, kAttnWarps * 32, smem, s>>>(*a);
  else grouped_attn_kernel<__nv_bfloat16><<<grid, kAttnWarps * 32, smem, s>>>(*a);
  return done();
}
