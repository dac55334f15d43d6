// Grouped-query attention: the row kernel between the projection and the attention kernels (norms, rotation, cache rows, query
// layout), the means of pooled blocks, and the plain attention kernel for sizes and types that the tensor-core kernels
// (attn_decode.cu, attn_prefill_umma.cu) do not cover.
#include <math_constants.h>

#include <type_traits>

#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"

namespace xpool {
namespace grouped {

using elem::ld;
using elem::st;

constexpr int kPrepThreads = 256;
constexpr int kAttnWarps = 4;

// N elements at a time: 16 bytes where the layouts allow it, else one.
template <int N, typename T>
__device__ __forceinline__ void load_n(const T* p, float (&v)[N]) {
  if constexpr (N == 8) {
    float lo[4], hi[4];
    const uint4 x = *reinterpret_cast<const uint4*>(p);
    const uint2 h[2] = {make_uint2(x.x, x.y), make_uint2(x.z, x.w)};
    elem::ldv<4>(reinterpret_cast<const T*>(&h[0]), lo);
    elem::ldv<4>(reinterpret_cast<const T*>(&h[1]), hi);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = lo[j], v[4 + j] = hi[j];
  } else {
    elem::ldv<N>(p, v);
  }
}
template <int N, typename T>
__device__ __forceinline__ void store_n(T* p, const float (&v)[N]) {
  if constexpr (N == 8) {
    float lo[4], hi[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) lo[j] = v[j], hi[j] = v[4 + j];
    uint2 h[2];
    elem::stv<4>(reinterpret_cast<T*>(&h[0]), lo);
    elem::stv<4>(reinterpret_cast<T*>(&h[1]), hi);
    *reinterpret_cast<uint4*>(p) = make_uint4(h[0].x, h[0].y, h[1].x, h[1].y);
  } else {
    elem::stv<N>(p, v);
  }
}

// N elements as they lie in memory.
template <typename T, int N>
struct alignas(N * sizeof(T)) Raw {
  T v[N];
};

// Row of a paged cache of `heads` heads of `width` elements.
__device__ __forceinline__ size_t paged_row(const int* table, int t, int page_size, int heads, int h, int width) {
  return ((static_cast<size_t>(table[t / page_size]) * page_size + t % page_size) * heads + h) * width;
}

// Mean of the `pool` cached rows that end with token `last`, elements c .. c + N - 1 of head h. `own`, where given, is what the
// cache holds for the last token. kFlight rows are in flight.
template <int N, int kFlight, typename T>
__device__ __forceinline__ void block_mean(const T* cache, const int* table, int last, int pool, int page_size, int heads, int h, int width, int c,
                                           const float* own, float (&mean)[N]) {
#pragma unroll
  for (int j = 0; j < N; ++j) mean[j] = 0.f;
  const int stop = own != nullptr ? last : last + 1;
  for (int t = last + 1 - pool; t < stop; t += kFlight) {
    float v[kFlight][N];
#pragma unroll
    for (int u = 0; u < kFlight; ++u) load_n<N>(cache + paged_row(table, min(t + u, stop - 1), page_size, heads, h, width) + c, v[u]);
#pragma unroll
    for (int u = 0; u < kFlight; ++u)
#pragma unroll
      for (int j = 0; j < N; ++j) mean[j] += t + u < stop ? v[u][j] : 0.f;
  }
#pragma unroll
  for (int j = 0; j < N; ++j) mean[j] = (own != nullptr ? mean[j] + own[j] : mean[j]) / static_cast<float>(pool);
}

// A CTA (or several, grid y) per row, L lanes per head slot: padded query heads, then keys, then values. A lane takes N elements at a time and the
// same columns of every slot it serves, so that it looks up their turns once; kAhead slots are in flight, and registers are kept
// for four CTAs of 256 threads. kInter: pairs of neighbours turn. kMeans: rows may complete blocks.
template <typename T, int N, int L, bool kInter, bool kMeans>
__global__ void __launch_bounds__(kPrepThreads, kMeans ? 2 : 4)
grouped_prep_kernel(XpGroupedPrepArgs a) {
  constexpr int kAhead = N == 1 ? 1 : kMeans ? 2 : 4;
  constexpr int kTurns = kInter && N > 1 ? N / 2 : N;
  const int per_row = a.kv_heads * (a.group_pad + 2), nq = a.kv_heads * a.group_pad, group = a.heads / a.kv_heads;
  const int row = blockIdx.x, lane = threadIdx.x % L, slots = blockDim.x / L * gridDim.y;   // slots at a time
  const T* proj = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.ld_proj;
  const int c0 = lane * N, rotated = 2 * a.rot_pairs;
  // first column of a slot in the row, -1: padding of a group
  auto column = [&](int u) {
    if (u < nq) {
      const int q = u / a.group_pad, g = u - q * a.group_pad;
      return g < group ? a.q_off + (q * group + g) * a.dim : -1;
    }
    const int h = u - nq;
    return h < a.kv_heads ? a.k_off + h * a.dim : a.v_off + (h - a.kv_heads) * a.vdim;
  };
  const int cache_row = a.slots[row];
  const int pos = a.positions != nullptr ? a.positions[row] : 0;
  const float2* turn = reinterpret_cast<const float2*>(a.rot) + static_cast<size_t>(pos < a.rot_positions ? pos : 0) * a.rot_pairs;
  auto pair_of = [&](int e) { return kInter ? e >> 1 : e >= a.rot_pairs ? e - a.rot_pairs : e; };
  float2 own_turn[kTurns];
#pragma unroll
  for (int j = 0; j < kTurns; ++j) {
    const int e = c0 + j * (N / kTurns);
    own_turn[j] = e < rotated ? turn[pair_of(e)] : make_float2(1.f, 0.f);
  }
  const bool means = kMeans && row < a.pool_rows && (pos + 1) % a.pool == 0;

  for (int u0 = blockIdx.y * (blockDim.x / L) + threadIdx.x / L; u0 < per_row + slots; u0 += slots * kAhead) {    // every lane of a warp takes part in the shuffles
    if (__all_sync(0xffffffffu, u0 >= per_row)) break;
    Raw<T, N> raw[kAhead];                           // the lane's first columns of every slot
#pragma unroll
    for (int k = 0; k < kAhead; ++k) {
      const int u = u0 + k * slots;
      const int at = u < per_row ? column(u) : -1;
      const bool some = at >= 0 && c0 < (u < nq + a.kv_heads ? a.dim : a.vdim);
      raw[k] = *reinterpret_cast<const Raw<T, N>*>(proj + (some ? at + c0 : a.q_off));      // no branch around the load
      if (!some) raw[k] = Raw<T, N>{};
    }
#pragma unroll
    for (int k = 0; k < kAhead; ++k) {
      const int u = u0 + k * slots;
      const bool qk = u < nq + a.kv_heads;
      const int at = u < per_row ? column(u) : -1;
      const T* src = proj + at;
      const int n = at < 0 ? 0 : qk ? a.dim : a.vdim, width = qk ? a.dq : a.dv;
      const float* weight = u < nq ? a.q_norm : a.k_norm;
      float inv = 1.f, x[N];
#pragma unroll
      for (int j = 0; j < N; ++j) x[j] = ld(&raw[k].v[j]);
      if (a.norm) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < N; ++j) ss += x[j] * x[j];
        for (int c = c0 + L * N; c < n; c += L * N) {
          float y[N];
          load_n<N>(src + c, y);
#pragma unroll
          for (int j = 0; j < N; ++j) ss += y[j] * y[j];
        }
#pragma unroll
        for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (qk && n > 0) inv = rsqrtf(ss / static_cast<float>(n) + a.eps);
      }
      if (u >= per_row || (u >= nq && cache_row < 0)) continue;
      T* dst;
      if (u < nq) {
        dst = reinterpret_cast<T*>(a.q_out) + (static_cast<size_t>(row) * nq + u) * a.dq;
      } else {
        const int h = u - nq - (qk ? 0 : a.kv_heads);
        dst = (qk ? reinterpret_cast<T*>(a.k_cache) : reinterpret_cast<T*>(a.v_cache)) + (static_cast<size_t>(cache_row) * a.kv_heads + h) * width;
      }
      for (int c = c0; c < width; c += L * N) {
        if (c != c0) {
#pragma unroll
          for (int j = 0; j < N; ++j) x[j] = 0.f;
          if (c < n) load_n<N>(src + c, x);
        }
        if (qk && c < n) {
#pragma unroll
          for (int j = 0; j < N; ++j) x[j] *= weight != nullptr ? inv * weight[c + j] : inv;
          if (c < rotated) {
            if constexpr (kInter && N > 1) {
#pragma unroll
              for (int j = 0; j < N; j += 2) {
                if (c + j >= rotated) continue;
                const float2 t = c == c0 ? own_turn[j / 2] : turn[(c + j) >> 1];
                const float v = x[j], w = x[j + 1];
                x[j] = v * t.x - w * t.y, x[j + 1] = w * t.x + v * t.y;
              }
            } else {
#pragma unroll
              for (int j = 0; j < N; ++j) {
                const int e = c + j;
                if (e >= rotated) continue;
                const bool second = kInter ? e & 1 : e >= a.rot_pairs;
                const int o = kInter ? e ^ 1 : second ? e - a.rot_pairs : e + a.rot_pairs;
                const float other = ld(src + o) * (weight != nullptr ? inv * weight[o] : inv);
                const float2 t = c == c0 ? own_turn[j] : turn[pair_of(e)];
                x[j] = second ? x[j] * t.x + other * t.y : x[j] * t.x - other * t.y;
              }
            }
          }
        }
        store_n<N>(dst + c, x);
        if (kMeans && means && u >= nq) {
          const int* table = a.block_table + static_cast<size_t>(row) * a.max_blocks;
          const int h = u - nq - (qk ? 0 : a.kv_heads);
          float own[N], mean[N];
          T held[N];
#pragma unroll
          for (int j = 0; j < N; ++j) st(&held[j], x[j]), own[j] = ld(&held[j]);
          block_mean<N, 4>(reinterpret_cast<const T*>(qk ? a.k_cache : a.v_cache), table, pos, a.pool, a.page_size, a.kv_heads, h, width, c, own, mean);
          store_n<N>(reinterpret_cast<T*>(qk ? a.k_pool : a.v_pool) + paged_row(table, pos / a.pool, a.pool_page, a.kv_heads, h, width) + c, mean);
        }
      }
    }
  }
}

// A CTA looks at kMeanRows rows, few of which complete a block.
constexpr int kMeanRows = 16;

template <typename T, int N>
__global__ void __launch_bounds__(kPrepThreads)
block_mean_kernel(XpBlockMeanArgs a) {
  const int first = blockIdx.x * kMeanRows, lane = threadIdx.x & 31;
  const int mine = first + (lane < kMeanRows ? lane : 0);
  const int my_pos = mine < a.rows ? a.positions[mine] : -1;
  const int my_seq = mine < a.rows && a.row_seq != nullptr ? a.row_seq[mine] : mine;
  const bool completes = lane < kMeanRows && my_pos >= 0 && a.slots[mine] >= 0 && (my_pos + 1) % a.pool == 0;
  const int nk = a.kv_heads * a.dq, total = nk + a.kv_heads * a.dv;
  for (uint32_t left = __ballot_sync(0xffffffffu, completes); left != 0; left &= left - 1) {
    const int from = __ffs(left) - 1, pos = __shfl_sync(0xffffffffu, my_pos, from), seq = __shfl_sync(0xffffffffu, my_seq, from);
    const int* table = a.block_table + static_cast<size_t>(seq) * a.max_blocks;
    for (int i = threadIdx.x * N; i < total; i += kPrepThreads * N) {
      const bool is_k = i < nk;
      const int width = is_k ? a.dq : a.dv, e = is_k ? i : i - nk, h = e / width, c = e % width;
      float mean[N];
      block_mean<N, 8>(reinterpret_cast<const T*>(is_k ? a.k_cache : a.v_cache), table, pos, a.pool, a.page_size, a.kv_heads, h, width, c, nullptr, mean);
      store_n<N>(reinterpret_cast<T*>(is_k ? a.k_pool : a.v_pool) + paged_row(table, pos / a.pool, a.pool_page, a.kv_heads, h, width) + c, mean);
    }
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
  // the kept first tokens (or the pooled blocks) in whole steps of 32, then the step in which the window begins and those behind it
  const int lo = a.window > 0 && len > a.window ? len - a.window : 0;
  const int blocks = a.pool > 0 ? lo / a.pool : 0;
  const int head = a.pool > 0 ? (blocks + 31) / 32 * 32 : min((a.keep_first + 31) / 32, lo / 32) * 32, skip = lo / 32 * 32 - head;
  const bool sig = a.sigmoid_bias != nullptr;
  const float bias = sig ? a.sigmoid_bias[h] : 0.f;
  float m = sig ? 0.f : -CUDART_INF_F, l = 0.f;
  for (int v0 = warp * 32; v0 + (v0 < head ? 0 : skip) < len; v0 += kAttnWarps * 32) {
    const bool pooled = a.pool > 0 && v0 < head;
    const int t0 = v0 + (v0 < head ? 0 : skip), t = t0 + lane, stop = pooled ? blocks : len;
    const bool on = t < stop && (pooled || t >= lo || t < a.keep_first);
    const int tt = t < stop ? t : t0;
    const size_t tok = paged_row(table, tt, pooled ? a.pool_page : a.page_size, a.kv_heads, hk, 1);
    const T* k = (pooled ? reinterpret_cast<const T*>(a.k_pool) : kc) + tok * a.dq;
    const T* vals = pooled ? reinterpret_cast<const T*>(a.v_pool) : vc;
    float s = 0.f;
    for (int c = 0; c < a.dim; ++c) s = fmaf(q_s[c], ld(k + c), s);
    if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
    if (!on) s = -CUDART_INF_F;
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float mn = sig ? 0.f : fmaxf(m, mx), corr = sig ? 1.f : m == -CUDART_INF_F ? 0.f : expf(m - mn);
    const float p = !on ? 0.f : sig ? elem::sigmoid(s + bias) : expf(s - mn);
    l = l * corr + elem::warp_sum(p);
    m = mn;
    const int live = min(32, stop - t0);
    for (int c = lane; c - lane < a.vdim; c += 32) {       // every lane takes part in the shuffles
      float v = c < a.vdim ? acc_s[c] * corr : 0.f;
      for (int j = 0; j < live; ++j) {
        const float pj = __shfl_sync(0xffffffffu, p, j);
        const size_t tj = __shfl_sync(0xffffffffu, static_cast<unsigned long long>(tok), j);
        if (c < a.vdim) v = fmaf(pj, ld(vals + tj * a.dv + c), v);
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
  if (a.sink != nullptr) {
    const float top = fmaxf(mm, a.sink[h]);
    ll = ll * expf(mm - top) + expf(a.sink[h] - top);
    mm = top;
  }
  float f = sig ? 1.f : 1.f / ll;
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
  if (a->rot_pairs < 0 || 2 * a->rot_pairs > a->dim || (a->rot_pairs > 0 && (a->rot == nullptr || a->rot_positions <= 0 || a->positions == nullptr))) return -12;
  if (a->pool > 0 && (a->pool_rows > a->rows || a->positions == nullptr || a->block_table == nullptr || a->k_pool == nullptr || a->v_pool == nullptr ||
                      a->pool_page <= 0 || a->page_size <= 0))
    return -13;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto al = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const int n = a->f32 ? 4 : 8;
  const bool v = a->dim % n == 0 && a->vdim % n == 0 && a->dq % n == 0 && a->dv % n == 0 && a->ld_proj % n == 0 && a->q_off % n == 0 && a->k_off % n == 0 &&
                 a->v_off % n == 0 && al(a->proj) && al(a->k_cache) && al(a->v_cache) && al(a->q_out) && al(a->k_pool) && al(a->v_pool);
  const int widest = a->dq > a->dv ? a->dq : a->dv;
  const int units = a->kv_heads * (a->group_pad + 2);
  auto run = [&](auto kernel, int lanes) {               // few rows: a slot per thread, four CTAs or more per row; many: four slots per thread
    const bool few = a->rows <= 512;
    const int want = few ? units * lanes : (units * lanes + 3) / 4, most = few ? 128 : kPrepThreads;
    const int threads = want < most ? (want + 31) / 32 * 32 : most;
    kernel<<<dim3(a->rows, few ? (want + threads - 1) / threads : 1), threads, 0, s>>>(*a);
  };
  auto pick = [&](auto inter, auto means) {
    constexpr bool I = decltype(inter)::value, M = decltype(means)::value;
    if (a->f32) {
      if (!v) run(grouped_prep_kernel<float, 1, 32, I, M>, 32);
      else if (widest <= 64) run(grouped_prep_kernel<float, 4, 16, I, M>, 16);
      else run(grouped_prep_kernel<float, 4, 32, I, M>, 32);
    } else {
      if (!v) run(grouped_prep_kernel<__nv_bfloat16, 1, 32, I, M>, 32);
      else if (widest <= 64) run(grouped_prep_kernel<__nv_bfloat16, 8, 8, I, M>, 8);
      else run(grouped_prep_kernel<__nv_bfloat16, 8, 16, I, M>, 16);
    }
  };
  const bool pooling = a->pool > 0 && a->pool_rows > 0;
  if (a->interleaved) pooling ? pick(std::true_type{}, std::true_type{}) : pick(std::true_type{}, std::false_type{});
  else pooling ? pick(std::false_type{}, std::true_type{}) : pick(std::false_type{}, std::false_type{});
  return done();
}

extern "C" int xp_block_mean(const XpBlockMeanArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->pool <= 0 || a->pool_page <= 0 || a->page_size <= 0 || a->kv_heads <= 0) return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto al = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const int n = a->f32 ? 4 : 8;
  const int blocks = (a->rows + kMeanRows - 1) / kMeanRows;
  const bool v = a->dq % n == 0 && a->dv % n == 0 && al(a->k_cache) && al(a->v_cache) && al(a->k_pool) && al(a->v_pool);
  if (a->f32) {
    if (v) block_mean_kernel<float, 4><<<blocks, kPrepThreads, 0, s>>>(*a);
    else block_mean_kernel<float, 1><<<blocks, kPrepThreads, 0, s>>>(*a);
  } else {
    if (v) block_mean_kernel<__nv_bfloat16, 8><<<blocks, kPrepThreads, 0, s>>>(*a);
    else block_mean_kernel<__nv_bfloat16, 1><<<blocks, kPrepThreads, 0, s>>>(*a);
  }
  return done();
}

extern "C" int xp_grouped_attn(const XpGroupedAttnArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->rows > 65535) return -10;
  if (a->pool > 0 && (a->window <= 0 || a->keep_first > 0 || a->pool_page <= 0 || a->k_pool == nullptr || a->v_pool == nullptr)) return -12;
  const size_t smem = static_cast<size_t>(a->dim + kAttnWarps * (a->vdim + 2)) * 4;
  if (smem > 48 * 1024) return -11;
  const dim3 grid(a->heads, a->rows);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->f32) grouped_attn_kernel<float><<<grid, kAttnWarps * 32, smem, s>>>(*a);
  else grouped_attn_kernel<__nv_bfloat16><<<grid, kAttnWarps * 32, smem, s>>>(*a);
  return done();
}
