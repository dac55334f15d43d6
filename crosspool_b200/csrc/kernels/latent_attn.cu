// Latent attention over a paged cache of [latent | rotated shared key] rows: one cache row per token serves every head,
// as key (all of it) and as value (its latent columns). Kernels:
//   latent_prep       per token: latent RMS norm, rotary on the shared key part and on every query head, cache write,
//                     query layouts of the two forms below
//   latent_attn_tc    absorbed form (queries already multiplied into the latent space), one token row and up to 32 heads
//                     per CTA, split over the sequence: a producer warp fills a ring of 64-token tiles; ldmatrix + mma.m16n8k16, the
//                     probabilities carried as a bf16 pair (high and low part). Bound by reading the cache once.
//   latent_attn_simt  the same in plain FMAs for any sizes and for fp32
//   latent_gather     dense copy of a sequence's cached rows, the input of the expanded form (keys and values per head,
//                     chunked prefill on the tcgen05 kernel of attn_prefill_umma.cu)
//
// mma.sync rather than tcgen05 in the absorbed decode kernel: a UMMA tile needs 64 or 128 query rows where there are 16 or 32.
// With tokens and latent columns on the M axis instead (heads on N), the fixed cost of the small-N instructions and the
// round trip of the scores through tensor memory made a tcgen05 form a third slower than this one.
#include <math_constants.h>

#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"
#include "xpool/sm100.cuh"

namespace xpool {
namespace latent {

constexpr float kLog2e = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------ prep
constexpr int kPrepThreads = 256;
constexpr int kPrepHeads = 8;              // heads per CTA (grid y): one per warp

template <typename T, int VEC>
__global__ void __launch_bounds__(kPrepThreads)
latent_prep_kernel(XpLatentPrepArgs a) {
  extern __shared__ float cs[];            // cos | sin, rot_dims / 2 each
  __shared__ float red[kPrepThreads / 32];
  const int row = blockIdx.x;
  const int half = a.rot_dims / 2;
  const T* proj = reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.ld_proj;
  const double pos = static_cast<double>(a.positions[row]);
  for (int i = threadIdx.x; i < half; i += kPrepThreads) {
    // the angle is reduced to one turn in double, so its fp32 sine and cosine are exact to fp32 at any position
    const double turns = pos * a.freq[i] * 0.15915494309189535;
    float s, c;
    sincospif(2.f * static_cast<float>(turns - rint(turns)), &s, &c);
    cs[i] = c;
    cs[half + i] = s;
  }
  __syncthreads();
  // element j of a vector x whose first rot_dims elements are rotated in pairs (j, j + half), or of neighbours
  auto rotated = [&](const T* x, int j) -> float {
    const float v = elem::ld(x + j);
    if (j >= a.rot_dims) return v;
    const bool first = a.interleaved ? (j & 1) == 0 : j < half;
    const int i = a.interleaved ? j >> 1 : first ? j : j - half;
    const float o = elem::ld(x + (a.interleaved ? j ^ 1 : first ? j + half : i));
    return first ? v * cs[i] - o * cs[half + i] : v * cs[i] + o * cs[half + i];
  };
  float q_inv = 1.f;                        // queries made from a latent lack its norm
  if (a.q_rank > 0) {
    float ss = 0.f;
    for (int c = threadIdx.x * VEC; c < a.q_rank; c += kPrepThreads * VEC) {
      float v[VEC];
      elem::ldv<VEC>(proj + a.ql_off + c, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss += v[j] * v[j];
    }
    q_inv = rsqrtf(elem::block_sum<kPrepThreads>(ss, red) / static_cast<float>(a.q_rank) + a.eps);
  }

  const int slot = a.slots[row];
  if (slot >= 0 && blockIdx.y == 0) {
    const T* kv = proj + a.kv_off;
    float ss = 0.f;
    for (int c = threadIdx.x; c < a.kv_rank; c += kPrepThreads) {
      const float v = elem::ld(kv + c);
      ss += v * v;
    }
    const float inv = rsqrtf(elem::block_sum<kPrepThreads>(ss, red) / static_cast<float>(a.kv_rank) + a.eps);
    T* dst = reinterpret_cast<T*>(a.cache) + static_cast<size_t>(slot) * a.ld_cache;
    for (int c = threadIdx.x; c < a.ld_cache; c += kPrepThreads) {
      float v = 0.f;                        // the pitch's padding columns hold zeros
      if (c < a.kv_rank) v = elem::ld(kv + c) * inv * a.norm_w[c];
      else if (c < a.kv_rank + a.rot) v = rotated(kv + a.kv_rank, c - a.kv_rank);
      elem::st(dst + c, v);
    }
  }

  // queries: one warp per head
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int dh = a.dim + a.rot;
  for (int h = blockIdx.y * kPrepHeads + warp; h < min(a.heads, static_cast<int>(blockIdx.y + 1) * kPrepHeads); h += kPrepThreads / 32) {
    const T* q = (a.q != nullptr ? reinterpret_cast<const T*>(a.q) + static_cast<size_t>(row) * a.ld_q : proj + a.q_off) + h * dh;
    T *plain, *rot;
    int plain_end, rot_end;                 // columns past the vector's own hold zeros
    if (row < a.abs_rows) {
      const size_t r = static_cast<size_t>(h) * a.qp_rows + row;
      plain = reinterpret_cast<T*>(a.q_plain) + r * a.dim_p;
      rot = reinterpret_cast<T*>(a.q_abs) + r * a.ld_abs + a.kv_rank;
      plain_end = a.dim_p;
      rot_end = a.ld_abs - a.kv_rank;
    } else {
      plain = reinterpret_cast<T*>(a.q_exp) + (static_cast<size_t>(row) * a.heads + h) * a.dq_pad;
      rot = plain + a.dim;
      plain_end = a.dim;
      rot_end = a.dq_pad - a.dim;
    }
    if (VEC == 4) {
      for (int c = lane * 4; c < a.dim; c += 128) {
        float v[4];
        elem::ldv<4>(q + c, v);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] *= q_inv;
        elem::stv<4>(plain + c, v);
      }
      for (int c = a.dim + lane; c < plain_end; c += 32) elem::st(plain + c, 0.f);
    } else {
      for (int c = lane; c < plain_end; c += 32) elem::st(plain + c, c < a.dim ? elem::ld(q + c) * q_inv : 0.f);
    }
    for (int c = lane; c < rot_end; c += 32) elem::st(rot + c, c < a.rot ? rotated(q + a.dim, c) * q_inv : 0.f);
  }
}

// ------------------------------------------------------------------------------------------ plain kernel
constexpr int kSimtThreads = 128;
constexpr int kSimtTile = 32;
constexpr int kSimtAcc = 8;              // latent columns per thread: kv_rank <= 1024

// First token that a row at the end of len tokens sees.
__device__ __forceinline__ int window_start(const XpLatentAttnArgs& a, int len) { return a.window > 0 ? max(0, len - a.window) : 0; }

template <typename T>
__global__ void __launch_bounds__(kSimtThreads)
latent_attn_simt_kernel(XpLatentAttnArgs a) {
  extern __shared__ float q_s[];         // kv_rank + rot
  __shared__ float sc[kSimtTile];
  const int h = blockIdx.x, row = blockIdx.y;
  const int dk = a.kv_rank + a.rot;
  T* out = reinterpret_cast<T*>(a.out) + (static_cast<size_t>(h) * a.q_rows + row) * a.ld_out;
  if (a.slots[row] < 0) {
    for (int c = threadIdx.x; c < a.kv_rank; c += kSimtThreads) elem::st(out + c, 0.f);
    return;
  }
  const T* q = reinterpret_cast<const T*>(a.q) + (static_cast<size_t>(h) * a.q_rows + row) * a.ld_q;
  for (int c = threadIdx.x; c < dk; c += kSimtThreads) q_s[c] = elem::ld(q + c) * a.scale * kLog2e;
  __syncthreads();
  const int* table = a.block_table + static_cast<size_t>(a.row_seq != nullptr ? a.row_seq[row] : row) * a.max_blocks;
  const T* cache = reinterpret_cast<const T*>(a.cache);
  const int len = a.positions[row] + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  auto token_row = [&](int t) {
    return cache + (static_cast<size_t>(table[t / a.page_size]) * a.page_size + t % a.page_size) * a.ld_cache;
  };
  float m = -CUDART_INF_F, l = 0.f, acc[kSimtAcc];
#pragma unroll
  for (int j = 0; j < kSimtAcc; ++j) acc[j] = 0.f;
  for (int t0 = window_start(a, len); t0 < len; t0 += kSimtTile) {
    const int n = min(kSimtTile, len - t0);
    for (int j = warp; j < n; j += kSimtThreads / 32) {
      const T* k = token_row(t0 + j);
      float s = 0.f;
      for (int c = lane; c < dk; c += 32) s = fmaf(q_s[c], elem::ld(k + c), s);
      s = elem::warp_sum(s);
      if (lane == 0) sc[j] = s;
    }
    __syncthreads();
    float mn = m;
    for (int j = 0; j < n; ++j) mn = fmaxf(mn, sc[j]);
    const float f = exp2f(m - mn);       // 0 on the first tile (m = -inf)
    m = mn;
    l *= f;
#pragma unroll
    for (int j = 0; j < kSimtAcc; ++j) acc[j] *= f;
    for (int j = 0; j < n; ++j) {
      const float p = exp2f(sc[j] - m);
      l += p;
      const T* v = token_row(t0 + j);
#pragma unroll
      for (int u = 0; u < kSimtAcc; ++u) {
        const int c = threadIdx.x + u * kSimtThreads;
        if (c < a.kv_rank) acc[u] = fmaf(p, elem::ld(v + c), acc[u]);
      }
    }
    __syncthreads();
  }
  float g = 1.f / l;
  if (a.gate != nullptr) g *= elem::sigmoid(elem::ld(reinterpret_cast<const T*>(a.gate) + static_cast<size_t>(row) * a.ld_gate + h));
#pragma unroll
  for (int u = 0; u < kSimtAcc; ++u) {
    const int c = threadIdx.x + u * kSimtThreads;
    if (c < a.kv_rank) elem::st(out + c, acc[u] * g);
  }
}

// ------------------------------------------------------------------------------------------ tensor-core kernel
constexpr int kTcWarps = 8;              // compute warps: 4 token groups x 2 halves of the key columns, then 8 column groups
constexpr int kTcThreads = kTcWarps * 32 + 32;   // and a producer warp
constexpr int kTablePages = 512;         // page-table entries of a slice kept in shared memory
constexpr int kTile = 64;                // tokens per tile
constexpr int kPPitch = kTile + 8;

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int V>
struct Count {
  static constexpr int value = V;
};

struct TcLayout {
  int pitch;        // elements of one shared-memory row (an odd multiple of 16 bytes: conflict-free ldmatrix)
  int stage_bytes;
  int q_bytes;
  int stages;
  int total;
};

__host__ __device__ inline TcLayout tc_layout(int dk16, int vcols, int hg) {
  TcLayout L;
  const int w = dk16 > vcols ? dk16 : vcols;
  L.pitch = w + 8;
  L.stage_bytes = kTile * L.pitch * 2;
  const int m = 16 * hg;
  L.q_bytes = m * L.pitch * 2;
  const int fixed = 128 + L.q_bytes + 2 * m * kPPitch * 2 + 2 * m * kTile * 4 + 3 * m * 4 + kTablePages * 4;
  int st = (100 * 1024 - fixed) / L.stage_bytes;     // two CTAs per SM when the rows are short
  if (st < 2) st = 2;
  if (st > 4) st = 4;
  L.stages = st;
  L.total = fixed + st * L.stage_bytes;
  return L;
}

__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes),
               "r"(bar)
               : "memory");
}

// Barrier of the compute warps; true when any of their threads passes true.
__device__ __forceinline__ bool compute_any(bool p) {
  uint32_t r;
  asm volatile(
      "{\n\t"
      ".reg .pred a, b;\n\t"
      "setp.ne.u32 a, %1, 0;\n\t"
      "barrier.cta.red.or.pred b, 1, %2, a;\n\t"
      "selp.u32 %0, 1, 0, b;\n\t"
      "}"
      : "=r"(r)
      : "r"(p ? 1u : 0u), "n"(kTcWarps * 32)
      : "memory");
  return r != 0;
}

// NT: 8-column tiles of the latent per warp (kv_rank <= 64 * NT). HG: groups of 16 heads that share a CTA's tiles.
// A producer warp keeps the ring of tiles full (one bulk copy per cached row), so that the compute warps meet at two
// barriers per tile only: behind the scores and behind the probabilities.
template <int NT, int HG>
__global__ void __launch_bounds__(kTcThreads)
latent_attn_tc_kernel(XpLatentAttnArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int MH = 16 * HG;                        // heads of the CTA
  const int split = blockIdx.x, h0 = blockIdx.y * MH, row = blockIdx.z;
  const int nh = min(MH, a.heads - h0);
  const int dk16 = a.ld_cache;
  const TcLayout L = tc_layout(dk16, 64 * NT, HG);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem);                                  // [4] tile landed
  uint64_t* empty = full + 4;                                                          // [4] tile consumed
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem + 128);
  __nv_bfloat16* p_s = q_s + L.q_bytes / 2;                                            // high parts, then low parts
  float* s_s = reinterpret_cast<float*>(p_s + 2 * MH * kPPitch);                       // [2][MH][kTile]
  float* m_s = s_s + 2 * MH * kTile;                                                   // final maximum and sum, tile's factor
  float* l_s = m_s + MH;
  float* f_s = l_s + MH;
  int* table_s = reinterpret_cast<int*>(f_s + MH);
  uint8_t* ring = smem + L.total - L.stages * L.stage_bytes;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool pad = a.slots[row] < 0;
  const int len = pad ? 0 : a.positions[row] + 1;
  const int chunk = a.chunk_tokens > 0 ? a.chunk_tokens : len;
  const int t0 = window_start(a, len) + split * chunk, t1 = a.num_splits > 1 ? min(len, t0 + chunk) : len;
  if (a.num_splits > 1 && t0 >= len) return;         // the merge kernel skips this slice
  const int tiles = (t1 - t0 + kTile - 1) / kTile;
  const int* table = a.block_table + static_cast<size_t>(a.row_seq != nullptr ? a.row_seq[row] : row) * a.max_blocks;
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(a.cache);
  const int chunks_row = dk16 / 8;                   // 16-byte pieces of a row

  if (threadIdx.x == 0) {
    for (int i = 0; i < L.stages; ++i) {
      sm100::mbar_init(&full[i], 1);
      sm100::mbar_init(&empty[i], kTcWarps);
    }
    sm100::mbar_fence_init();
    sm100::fence_proxy_async_smem();
  }
  // the slice's page table, so that no copy waits for a lookup in memory
  const int page0 = t0 / a.page_size, pages = tiles > 0 ? (t1 - 1) / a.page_size - page0 + 1 : 0;
  const bool cached = pages <= kTablePages;
  if (cached)
    for (int i = threadIdx.x; i < pages; i += kTcThreads) table_s[i] = table[page0 + i];
  __syncthreads();

  if (warp == kTcWarps) {
    for (int it = 0; it < tiles; ++it) {
      const int b = it % L.stages, n = min(kTile, t1 - t0 - it * kTile);
      if (it >= L.stages) {
        const uint32_t parity = ((it / L.stages) - 1) & 1;
        const bool ok = sm100::mbar_try_wait(&empty[b], parity) ||
                        sm100::mbar_wait(&empty[b], parity, sm100::global_timer_ns() + sm100::kPipelineWaitNs);
        if (!__all_sync(0xffffffffu, ok)) break;       // the compute warps' own wait runs out and reports it
      }
      uint8_t* st = ring + b * L.stage_bytes;
      // rows past the slice: zeros (their probability is zero, but not their memory); this is the last tile
      for (int i = lane; i < (kTile - n) * chunks_row; i += 32)
        *reinterpret_cast<uint4*>(st + (n + i / chunks_row) * L.pitch * 2 + (i % chunks_row) * 16) = make_uint4(0, 0, 0, 0);
      __syncwarp();
      const uint32_t bar = sm100::smem_u32(&full[b]);
      if (lane == 0) sm100::mbar_arrive_expect_tx_addr(bar, static_cast<uint32_t>(n * dk16 * 2));
      __syncwarp();
      for (int tok = lane; tok < n; tok += 32) {
        const int t = t0 + it * kTile + tok, page = t / a.page_size;
        const __nv_bfloat16* src =
            cache + (static_cast<size_t>(cached ? table_s[page - page0] : table[page]) * a.page_size + (t - page * a.page_size)) * dk16;
        bulk_load(sm100::smem_u32(st + tok * L.pitch * 2), src, static_cast<uint32_t>(dk16 * 2), bar);
      }
    }
    return;
  }

  // queries of the head groups; absent heads read as zero
  for (int i = threadIdx.x; i < MH * chunks_row; i += kTcWarps * 32) {
    const int h = i / chunks_row, c = (i - h * chunks_row) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (h < nh)
      v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(a.q) +
                                          (static_cast<size_t>(h0 + h) * a.q_rows + row) * a.ld_q + c);
    *reinterpret_cast<uint4*>(q_s + h * L.pitch + c) = v;
  }
  const float qscale = a.scale * kLog2e;
  const int tg = warp & 3, kh = warp >> 2;           // token group (16 tokens), half of the key columns
  const int ksteps = dk16 / 16, ks0 = kh ? (ksteps + 1) / 2 : 0, ks1 = kh ? ksteps : (ksteps + 1) / 2;
  const int g = lane >> 2, q4 = lane & 3;
  const uint32_t q_addr = sm100::smem_u32(q_s) + ((lane & 15) * L.pitch + (lane >> 4) * 8) * 2;
  const uint32_t q_group = 16 * L.pitch * 2;
  const uint32_t k_lane = ((tg * 16 + (lane & 7) + ((lane >> 4) << 3)) * L.pitch + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t p_addr = sm100::smem_u32(p_s) + ((lane & 15) * kPPitch + (lane >> 4) * 8) * 2;
  const uint32_t v_lane = (((lane & 7) + ((lane >> 3) & 1) * 8) * L.pitch + warp * NT * 8 + (lane >> 4) * 8) * 2;
  constexpr int MW = MH / 8;                         // heads whose softmax this warp does: warp * MW ..
  float m_run[MW], l_run[MW];
#pragma unroll
  for (int r = 0; r < MW; ++r) m_run[r] = -CUDART_INF_F, l_run[r] = 0.f;
  float acc[HG][NT][4];
#pragma unroll
  for (int hg = 0; hg < HG; ++hg)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[hg][j][e] = 0.f;

  bool failed = false;
  compute_any(false);                                // queries are in place
  for (int it = 0; it < tiles; ++it) {
    const int b = it % L.stages;
    const uint32_t parity = (it / L.stages) & 1;
    const bool ok = sm100::mbar_try_wait(&full[b], parity) ||
                    sm100::mbar_wait(&full[b], parity, sm100::global_timer_ns() + sm100::kPipelineWaitNs);
    const uint32_t st = sm100::smem_u32(ring + b * L.stage_bytes);
    // scores of 16 tokens over this warp's half of the columns; even and odd steps in chains of their own
    float sc[2][HG][2][4];
#pragma unroll
    for (int i = 0; i < 2 * HG * 2 * 4; ++i) (&sc[0][0][0][0])[i] = 0.f;
    // kGroup steps at a time: all their fragments are requested before the first product
    auto score_steps = [&](int ks, auto count) {
      constexpr int kGroup = decltype(count)::value;
      uint32_t kb[kGroup][4], qa[kGroup][HG][4];
#pragma unroll
      for (int i = 0; i < kGroup; ++i) {
        ldsm_x4(st + k_lane + (ks + i) * 32, kb[i]);
#pragma unroll
        for (int hg = 0; hg < HG; ++hg) ldsm_x4(q_addr + hg * q_group + (ks + i) * 32, qa[i][hg]);
      }
#pragma unroll
      for (int i = 0; i < kGroup; ++i)
#pragma unroll
        for (int hg = 0; hg < HG; ++hg) {
          mma16816(sc[i & 1][hg][0], qa[i][hg], kb[i][0], kb[i][1]);
          mma16816(sc[i & 1][hg][1], qa[i][hg], kb[i][2], kb[i][3]);
        }
    };
    int ks = ks0;
    for (; ks + 6 <= ks1; ks += 6) score_steps(ks, Count<6>{});
    for (; ks + 2 <= ks1; ks += 2) score_steps(ks, Count<2>{});
    if (ks < ks1) score_steps(ks, Count<1>{});
#pragma unroll
    for (int hg = 0; hg < HG; ++hg)
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          *reinterpret_cast<float2*>(s_s + (kh * MH + hg * 16 + g + r * 8) * kTile + tg * 16 + u * 8 + q4 * 2) =
              make_float2(sc[0][hg][u][2 * r] + sc[1][hg][u][2 * r], sc[0][hg][u][2 * r + 1] + sc[1][hg][u][2 * r + 1]);
    failed = compute_any(!ok);
    if (failed) break;
    // softmax: MW heads per warp (independent chains), two tokens per lane
    const int tok0 = t0 + it * kTile + lane * 2;
    float v[MW][2], mx[MW], sum[MW];
#pragma unroll
    for (int r = 0; r < MW; ++r) {
      const int h = warp * MW + r;
      const float2 x = *reinterpret_cast<const float2*>(s_s + h * kTile + lane * 2);
      const float2 y = *reinterpret_cast<const float2*>(s_s + (MH + h) * kTile + lane * 2);
      v[r][0] = tok0 < t1 ? (x.x + y.x) * qscale : -CUDART_INF_F;
      v[r][1] = tok0 + 1 < t1 ? (x.y + y.y) * qscale : -CUDART_INF_F;
      mx[r] = fmaxf(v[r][0], v[r][1]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int r = 0; r < MW; ++r) mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], o));
#pragma unroll
    for (int r = 0; r < MW; ++r) {
      const int h = warp * MW + r;
      const float m_new = fmaxf(m_run[r], mx[r]);
      const float p0 = exp2f(v[r][0] - m_new), p1 = exp2f(v[r][1] - m_new);
      const float f = exp2f(m_run[r] - m_new);
      m_run[r] = m_new;
      l_run[r] *= f;
      sum[r] = p0 + p1;
      const __nv_bfloat162 hi = __floats2bfloat162_rn(p0, p1);
      const float2 hf = __bfloat1622float2(hi);
      *reinterpret_cast<__nv_bfloat162*>(p_s + h * kPPitch + lane * 2) = hi;
      *reinterpret_cast<__nv_bfloat162*>(p_s + (MH + h) * kPPitch + lane * 2) = __floats2bfloat162_rn(p0 - hf.x, p1 - hf.y);
      if (lane == 0) f_s[h] = f;
    }
    compute_any(false);
    // the sums are off the critical path: their shuffles overlap the second product
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int r = 0; r < MW; ++r) sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], o);
#pragma unroll
    for (int r = 0; r < MW; ++r) l_run[r] += sum[r];
#pragma unroll
    for (int hg = 0; hg < HG; ++hg) {
      const float fa = f_s[hg * 16 + g], fb = f_s[hg * 16 + g + 8];
#pragma unroll
      for (int j = 0; j < NT; ++j) acc[hg][j][0] *= fa, acc[hg][j][1] *= fa, acc[hg][j][2] *= fb, acc[hg][j][3] *= fb;
    }
#pragma unroll
    for (int kk = 0; kk < kTile / 16; ++kk) {
      uint32_t ph[HG][4], pl[HG][4];
#pragma unroll
      for (int hg = 0; hg < HG; ++hg) {
        ldsm_x4(p_addr + hg * 16 * kPPitch * 2 + kk * 32, ph[hg]);
        ldsm_x4(p_addr + (MH + hg * 16) * kPPitch * 2 + kk * 32, pl[hg]);
      }
      uint32_t vb[NT / 2][4];
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) ldsm_x4_trans(st + v_lane + kk * 16 * L.pitch * 2 + j * 32, vb[j]);
      // high parts of every column tile, then low parts: products on one accumulator stay far apart
#pragma unroll
      for (int hg = 0; hg < HG; ++hg)
#pragma unroll
        for (int j = 0; j < NT; ++j) mma16816(acc[hg][j], ph[hg], vb[j / 2][(j & 1) * 2], vb[j / 2][(j & 1) * 2 + 1]);
#pragma unroll
      for (int hg = 0; hg < HG; ++hg)
#pragma unroll
        for (int j = 0; j < NT; ++j) mma16816(acc[hg][j], pl[hg], vb[j / 2][(j & 1) * 2], vb[j / 2][(j & 1) * 2 + 1]);
    }
    __syncwarp();
    if (lane == 0) sm100::mbar_arrive(&empty[b]);
  }
  if (failed) {
    if (threadIdx.x == 0 && a.status != nullptr) atomicCAS(a.status, 0u, 8u);
    __nanosleep(1000000);   // copies still in flight get a bounded chance to land before the CTA retires
    return;
  }
#pragma unroll
  for (int r = 0; r < MW; ++r)
    if (lane == 0) {
      m_s[warp * MW + r] = m_run[r];
      l_s[warp * MW + r] = l_run[r];
    }
  compute_any(false);
#pragma unroll
  for (int hg = 0; hg < HG; ++hg)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int h = hg * 16 + g + e * 8;
      if (h >= nh) continue;
      if (a.num_splits > 1) {
        float* w = a.ws + ((static_cast<size_t>(row) * a.heads + h0 + h) * a.num_splits + split) * (a.kv_rank + 2);
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const int c = (warp * NT + j) * 8 + q4 * 2;
#pragma unroll
          for (int u = 0; u < 2; ++u)
            if (c + u < a.kv_rank) w[c + u] = acc[hg][j][e * 2 + u];
        }
        if (warp == 0 && q4 == 0) {
          w[a.kv_rank] = m_s[h];
          w[a.kv_rank + 1] = l_s[h];
        }
      } else {
        float f = pad ? 0.f : 1.f / l_s[h];
        if (a.gate != nullptr)
          f *= elem::sigmoid(elem::ld(reinterpret_cast<const __nv_bfloat16*>(a.gate) + static_cast<size_t>(row) * a.ld_gate + h0 + h));
        __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (static_cast<size_t>(h0 + h) * a.q_rows + row) * a.ld_out;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const int c = (warp * NT + j) * 8 + q4 * 2;
          if (c + 1 < a.kv_rank && a.ld_out % 2 == 0) {
            *reinterpret_cast<__nv_bfloat162*>(out + c) = __floats2bfloat162_rn(acc[hg][j][e * 2] * f, acc[hg][j][e * 2 + 1] * f);
          } else {
#pragma unroll
            for (int u = 0; u < 2; ++u)
              if (c + u < a.kv_rank) out[c + u] = __float2bfloat16_rn(acc[hg][j][e * 2 + u] * f);
          }
        }
      }
    }
}

constexpr int kMaxSlices = 64;

// One CTA per (head, row): folds the slices in order.
__global__ void __launch_bounds__(128)
latent_merge_kernel(XpLatentAttnArgs a) {
  const int h = blockIdx.x, row = blockIdx.y;
  const bool pad = a.slots[row] < 0;
  const int len = pad ? 0 : a.positions[row] + 1;
  const int n = min(a.num_splits, (len - window_start(a, len) + a.chunk_tokens - 1) / a.chunk_tokens);
  const int step = a.kv_rank + 2;
  const float* w = a.ws + (static_cast<size_t>(row) * a.heads + h) * a.num_splits * step;
  // the slices' maxima and sums, a slice per lane; every warp computes the same factors
  __shared__ float scale_s[kMaxSlices];
  const int lane = threadIdx.x & 31;
  float ms[kMaxSlices / 32], ls[kMaxSlices / 32], m = -CUDART_INF_F, l = 0.f;
#pragma unroll
  for (int i = 0; i < kMaxSlices / 32; ++i) {
    const int s = lane + 32 * i;
    ms[i] = s < n ? w[s * step + a.kv_rank] : -CUDART_INF_F;
    ls[i] = s < n ? w[s * step + a.kv_rank + 1] : 0.f;
    m = fmaxf(m, ms[i]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
#pragma unroll
  for (int i = 0; i < kMaxSlices / 32; ++i) {
    const float c = ms[i] == -CUDART_INF_F ? 0.f : exp2f(ms[i] - m);
    l += ls[i] * c;
    if (threadIdx.x < 32) scale_s[lane + 32 * i] = c;
  }
  l = elem::warp_sum(l);
  float f = pad ? 0.f : 1.f / l;
  __syncthreads();
  if (a.gate != nullptr)
    f *= elem::sigmoid(elem::ld(reinterpret_cast<const __nv_bfloat16*>(a.gate) + static_cast<size_t>(row) * a.ld_gate + h));
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (static_cast<size_t>(h) * a.q_rows + row) * a.ld_out;
  for (int c = threadIdx.x; c < a.kv_rank; c += 128) {
    float v = 0.f;
    for (int s0 = 0; s0 < n; s0 += 8) {              // eight slices in flight
      float x[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) x[u] = w[min(s0 + u, n - 1) * step + c];
#pragma unroll
      for (int u = 0; u < 8; ++u) v += s0 + u < n ? x[u] * scale_s[s0 + u] : 0.f;
    }
    out[c] = __float2bfloat16_rn(v * f);
  }
}

// ------------------------------------------------------------------------------------------ gather
constexpr int kGatherTokens = 4;

__global__ void __launch_bounds__(128)
latent_gather_kernel(XpLatentGatherArgs a) {
  const int seq = blockIdx.y;
  const int ctx = a.ctx_lens[seq], base = a.window > 0 ? max(0, ctx - a.window + 1) & ~63 : 0;
  const int len = ctx + a.q_lens[seq] - base;
  const int row_bytes = a.ld_cache * a.elem_bytes;   // a multiple of 16
  const int* table = a.block_table + static_cast<size_t>(seq) * a.max_blocks;
  const uint8_t* cache = static_cast<const uint8_t*>(a.cache);
  uint8_t* out = static_cast<uint8_t*>(a.out) + static_cast<size_t>(a.starts[seq]) * row_bytes;
  const int per = row_bytes / 16;
  const int t0 = blockIdx.x * kGatherTokens, n = min(kGatherTokens, len - t0);
  for (int u = threadIdx.x; u < n * per; u += 128) {
    const int t = t0 + u / per, c = u % per, from = base + t;
    const size_t src = (static_cast<size_t>(table[from / a.page_size]) * a.page_size + from % a.page_size) * row_bytes;
    *reinterpret_cast<uint4*>(out + static_cast<size_t>(t) * row_bytes + c * 16) =
        __ldg(reinterpret_cast<const uint4*>(cache + src + c * 16));
  }
}

inline int done() {
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -100 - static_cast<int>(e);
}

template <int NT, int HG>
int launch_tc(const XpLatentAttnArgs& a, cudaStream_t s) {
  const TcLayout L = tc_layout(a.ld_cache, 64 * NT, HG);
  if (L.total > 227 * 1024) return 1;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(latent_attn_tc_kernel<NT, HG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -21;
    set = true;
  }
  dim3 grid(a.num_splits > 1 ? a.num_splits : 1, (a.heads + 16 * HG - 1) / (16 * HG), a.rows);
  latent_attn_tc_kernel<NT, HG><<<grid, kTcThreads, L.total, s>>>(a);
  if (a.num_splits > 1) latent_merge_kernel<<<dim3(a.heads, a.rows), 128, 0, s>>>(a);
  return done();
}

}  // namespace latent
}  // namespace xpool

using namespace xpool::latent;

extern "C" int xp_latent_prep(const XpLatentPrepArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->rot_dims % 2 != 0 || a->rot_dims > a->rot || a->rot_dims > 2048 || a->ld_cache < a->kv_rank + a->rot) return -10;
  if (a->abs_rows > 0 && (a->q_plain == nullptr || a->q_abs == nullptr || a->ld_abs < a->kv_rank + a->rot || a->abs_rows > a->qp_rows ||
                          a->dim_p < a->dim))
    return -11;
  if (a->q == nullptr ? a->q_rank > 0 : a->ld_q < a->heads * (a->dim + a->rot)) return -13;
  if (a->abs_rows < a->rows && (a->q_exp == nullptr || a->dq_pad < a->dim + a->rot)) return -12;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const size_t sm = static_cast<size_t>(a->rot_dims > 0 ? a->rot_dims : 1) * 4;
  // four elements at a time where every head's plain part starts on a 4-element boundary in all layouts
  const int eb = a->f32 ? 4 : 2;
  auto al = [&](const void* p) { return reinterpret_cast<uintptr_t>(p) % (4 * eb) == 0; };
  const bool v = a->dim % 4 == 0 && a->rot % 4 == 0 && a->ld_proj % 4 == 0 && a->q_off % 4 == 0 && a->dim_p % 4 == 0 && a->dq_pad % 4 == 0 &&
                 al(a->proj) && al(a->q_plain) && al(a->q_exp) && al(a->q) && a->ld_q % 4 == 0 && a->q_rank % 4 == 0 && a->ql_off % 4 == 0;
  dim3 grid(a->rows, (a->heads + kPrepHeads - 1) / kPrepHeads);
  if (a->f32) {
    if (v) latent_prep_kernel<float, 4><<<grid, kPrepThreads, sm, s>>>(*a);
    else latent_prep_kernel<float, 1><<<grid, kPrepThreads, sm, s>>>(*a);
  } else {
    if (v) latent_prep_kernel<__nv_bfloat16, 4><<<grid, kPrepThreads, sm, s>>>(*a);
    else latent_prep_kernel<__nv_bfloat16, 1><<<grid, kPrepThreads, sm, s>>>(*a);
  }
  return done();
}

extern "C" int xp_latent_attn(const XpLatentAttnArgs* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->heads <= 0 || a->kv_rank <= 0 || a->page_size <= 0 || a->rows > a->q_rows || a->ld_q < a->kv_rank + a->rot) return -10;
  if (a->num_splits > 1 && (a->ws == nullptr || a->chunk_tokens <= 0 || a->num_splits > kMaxSlices)) return -11;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (!a->f32 && !a->force_simt && a->kv_rank <= 512 && a->ld_cache % 16 == 0 && a->ld_q % 8 == 0 && a->ld_q >= a->ld_cache) {
    int rc;
    if (a->heads > 16) rc = a->kv_rank <= 128 ? launch_tc<2, 2>(*a, s) : a->kv_rank <= 256 ? launch_tc<4, 2>(*a, s) : launch_tc<8, 2>(*a, s);
    else rc = a->kv_rank <= 128 ? launch_tc<2, 1>(*a, s) : a->kv_rank <= 256 ? launch_tc<4, 1>(*a, s) : launch_tc<8, 1>(*a, s);
    if (rc <= 0) return rc;
  }
  if (a->kv_rank > kSimtAcc * kSimtThreads || a->kv_rank + a->rot > 12000) return -12;
  dim3 grid(a->heads, a->rows);
  const size_t sm = static_cast<size_t>(a->kv_rank + a->rot) * 4;
  if (a->f32) latent_attn_simt_kernel<float><<<grid, kSimtThreads, sm, s>>>(*a);
  else latent_attn_simt_kernel<__nv_bfloat16><<<grid, kSimtThreads, sm, s>>>(*a);
  return done();
}

extern "C" int xp_latent_gather(const XpLatentGatherArgs* a, void* stream) {
  if (a->n_seqs <= 0 || a->max_len <= 0) return 0;
  if ((a->ld_cache * a->elem_bytes) % 16 != 0) return -10;
  dim3 grid((a->max_len + kGatherTokens - 1) / kGatherTokens, a->n_seqs);
  latent_gather_kernel<<<grid, 128, 0, reinterpret_cast<cudaStream_t>(stream)>>>(*a);
  return done();
}
