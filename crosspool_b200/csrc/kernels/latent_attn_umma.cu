// Latent attention of single rows on the tcgen05 tensor cores: the absorbed form of latent_attn.cu (queries in the latent
// space, one cache row per token that is key and value of every head) with the TOKENS and the LATENT COLUMNS on the tensor
// core's M axis and the heads on its N axis, so that 16 or 32 heads cost what one costs and the kernel is bound by reading
// the cache once:
//   S^T [64 tokens x heads]   = K [tokens x columns] Q^T         A = the cache tile as it lands, K-major
//   O^T [columns x heads]    += V^T [columns x tokens] P^T       A = the same tile through an MN-major descriptor
// (mma.sync computes the same with the heads on M at a rate that leaves it bound by the tensor pipe.)
//
// One CTA serves up to 32 heads of one row over one slice of the sequence.
//   warps 0-3   softmax: two of them read S^T (thread = token) and pass it through shared memory; each warp then owns a
//               quarter of the heads (two tokens per lane), keeps their running maximum and sum, and writes P^T as a bf16
//               pair (high and low part) into swizzled shared memory. O^T is rescaled in tensor memory only when a
//               maximum grew by more than 2^8. At the end thread = latent column: normalise, gate, store.
//   warp 4      TMA producer: the query heads once, then a ring of 64-token tiles through the page table
//   warp 5      allocates tensor memory and issues every tcgen05.mma from one thread; S^T one tile ahead of O^T
// A tile's scores use M = 128 although it holds 64 tokens: the upper 64 rows read whatever follows the block in shared
// memory and give rows that nobody looks at, which costs nothing (the instruction's time is set by its fixed cost here).
// Every wait is bounded; one that runs out sets the abort word and the status word (8) and ends the CTA after a common
// barrier that frees the tensor memory.
#include <math_constants.h>

#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"
#include "xpool/sm100.cuh"
#include "xpool/tensormap.hpp"

namespace xpool {
namespace latent5 {

constexpr int kTile = 64;              // tokens per tile
constexpr int kBlock = kTile * 128;    // bytes of 64 columns of a tile
constexpr int kMaxStages = 4;
constexpr int kThreads = 192;
constexpr int kMaxDynamic = 225 * 1024;   // beside the static barriers
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kRescaleStep = 8.0f;   // log2 units

struct __align__(8) Bars {
  uint64_t q_full;
  uint64_t kv_full[kMaxStages];
  uint64_t kv_empty[kMaxStages];
  uint64_t s_full[2];
  uint64_t p_full;
  uint64_t pv_done;
  uint32_t tmem_base;
  volatile uint32_t abort_flag;
};

struct Layout {
  int blocks;        // 64-column blocks of a cache row
  int stages;
  int total;         // dynamic shared memory
};

// ring | queries [blocks][N rows of 128 bytes] | P^T high, low [N rows of 128 bytes] | scores [N][64] fp32
__host__ __device__ inline Layout layout(int width, int n) {
  Layout L;
  L.blocks = (width + 63) / 64;
  const int fixed = 1024 + L.blocks * n * 128 + 2 * n * 128 + n * kTile * 4;
  int st = (112 * 1024 - fixed) / (L.blocks * kBlock);       // two CTAs per SM when the rows are short
  if (st < 2) st = 2;
  if (st > kMaxStages) st = kMaxStages;
  L.stages = st;
  L.total = fixed + st * L.blocks * kBlock;
  return L;
}

__device__ __forceinline__ bool wait_bar(uint64_t* bar, uint32_t parity, Bars* b, uint32_t site) {
  if (sm100::mbar_try_wait(bar, parity)) return true;
  const uint64_t deadline = sm100::global_timer_ns() + sm100::kPipelineWaitNs;
  uint32_t spins = 0;
  while (!sm100::mbar_try_wait(bar, parity)) {
    if ((++spins & 0xffu) == 0) {
      if (b->abort_flag != 0) return false;
      if (sm100::global_timer_ns() > deadline) {
        b->abort_flag = site;
        return false;
      }
    }
  }
  return true;
}

// Barrier of the four softmax warps; true when any of their threads passes true.
__device__ __forceinline__ bool softmax_any(bool p) {
  uint32_t r;
  asm volatile(
      "{\n\t"
      ".reg .pred a, b;\n\t"
      "setp.ne.u32 a, %1, 0;\n\t"
      "barrier.cta.red.or.pred b, 1, 128, a;\n\t"
      "selp.u32 %0, 1, 0, b;\n\t"
      "}"
      : "=r"(r)
      : "r"(p ? 1u : 0u)
      : "memory");
  return r != 0;
}

// kind::f16 instruction descriptor, bf16 inputs, fp32 accumulate, A MN-major (bit 15), B K-major.
__host__ __device__ constexpr uint32_t idesc_a_mn(uint32_t m, uint32_t n) {
  return sm100::umma_idesc_bf16(m, n) | (1u << 15);
}

template <int N>
__device__ __forceinline__ void tmem_ld_n(uint32_t addr, uint32_t (&v)[32]) {
  if constexpr (N == 32) {
    sm100::tmem_ld32_issue(addr, v);
    sm100::tmem_ld_wait_all(v);
  } else {
    float f[16];
    sm100::tmem_ld16(addr, f);
#pragma unroll
    for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(f[i]);
  }
}

// N: heads of the CTA (16 or 32).
template <int N>
__global__ void __launch_bounds__(kThreads)
latent_attn_umma_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv, XpLatentAttnArgs a,
                        int box_tokens) {
  extern __shared__ uint8_t smem_dyn[];
  __shared__ Bars bars;
  __shared__ float f_s[N], m_s[N], l_s[N];
  __shared__ uint32_t r_s[4];
  constexpr uint32_t kTmemCols = N == 32 ? 256 : 128;
  constexpr uint32_t kOCol = 2 * N;                  // S^T buffers first, then O^T: one N-column block per 128 latent columns
  constexpr int kHeads = N / 4;                      // heads of a softmax warp
  const int split = blockIdx.x, h0 = blockIdx.y * N, row = blockIdx.z;
  const int nh = min(N, a.heads - h0);
  const bool pad = a.slots[row] < 0;
  const int len = pad ? 0 : a.positions[row] + 1;
  const int t0 = a.num_splits > 1 ? split * a.chunk_tokens : 0;
  const int t1 = a.num_splits > 1 ? min(len, t0 + a.chunk_tokens) : len;
  if (a.num_splits > 1 && t0 >= len) return;         // the merge kernel skips this slice
  const int tiles = (t1 - t0 + kTile - 1) / kTile;   // 0 for a padding row
  const Layout L = layout(a.ld_cache, N);
  const int blocks = L.blocks, stages = L.stages;
  const int mblocks = (a.kv_rank + 127) / 128;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t base = (sm100::smem_u32(smem_dyn) + 1023u) & ~1023u;
  const uint32_t stage_bytes = static_cast<uint32_t>(blocks) * kBlock;
  const uint32_t q_s = base + stages * stage_bytes, p_s = q_s + blocks * N * 128;
  float* s_s = reinterpret_cast<float*>(smem_dyn + (p_s + 2 * N * 128 - sm100::smem_u32(smem_dyn)));

  if (threadIdx.x == 0) {
    sm100::mbar_init(&bars.q_full, 1);
    for (int s = 0; s < kMaxStages; ++s) {
      sm100::mbar_init(&bars.kv_full[s], 1);
      sm100::mbar_init(&bars.kv_empty[s], 1);
    }
    sm100::mbar_init(&bars.s_full[0], 1);
    sm100::mbar_init(&bars.s_full[1], 1);
    sm100::mbar_init(&bars.p_full, 4);
    sm100::mbar_init(&bars.pv_done, 1);
    bars.abort_flag = 0;
    sm100::mbar_fence_init();
    sm100::fence_proxy_async_smem();
  }
  if (warp == 5) {
    sm100::tmem_alloc(&bars.tmem_base, kTmemCols);
    sm100::tmem_relinquish();
  }
  sm100::tc_fence_before_sync();
  __syncthreads();
  sm100::tc_fence_after_sync();
  const uint32_t tmem = bars.tmem_base;

  if (warp == 4 && tiles > 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      sm100::tma_prefetch_desc(&tmap_q);
      sm100::tma_prefetch_desc(&tmap_kv);
      sm100::mbar_arrive_expect_tx(&bars.q_full, static_cast<uint32_t>(blocks * N * 128));
    }
    __syncwarp();
    for (int b = lane; b < blocks; b += 32)
      sm100::tma_load_3d_addr(q_s + b * N * 128, &tmap_q, sm100::smem_u32(&bars.q_full), b * 64, row, h0);
    const int* table = a.block_table + static_cast<size_t>(a.row_seq != nullptr ? a.row_seq[row] : row) * a.max_blocks;
    const int boxes = kTile / box_tokens;
    for (int t = 0; t < tiles; ++t) {
      const int s = t % stages;
      if (t >= stages && !__all_sync(0xffffffffu, wait_bar(&bars.kv_empty[s], ((t / stages) - 1) & 1, &bars, 1))) break;
      if (lane == 0) sm100::mbar_arrive_expect_tx(&bars.kv_full[s], stage_bytes);
      __syncwarp();
      for (int i = lane; i < blocks * boxes; i += 32) {
        const int b = i / boxes, j = i - b * boxes;
        int tk = t0 + t * kTile + j * box_tokens;
        if (tk >= t1) tk = (t1 - 1) / box_tokens * box_tokens;   // boxes past the end repeat the last one (masked)
        const int tok = table[tk / a.page_size] * a.page_size + tk % a.page_size;
        sm100::tma_load_2d_addr(base + s * stage_bytes + b * kBlock + j * box_tokens * 128, reinterpret_cast<uint64_t>(&tmap_kv),
                                sm100::smem_u32(&bars.kv_full[s]), b * 64, tok, sm100::l2_policy_evict_normal());
      }
    }
  } else if (warp == 5 && tiles > 0) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      const uint32_t idesc_s = sm100::umma_idesc_bf16(128, N), idesc_o = idesc_a_mn(128, N);
      const int ksteps = (a.kv_rank + a.rot + 15) / 16;
      auto issue_s = [&](int t) {
        const uint32_t st = base + (t % stages) * stage_bytes, d = tmem + static_cast<uint32_t>((t & 1) * N);
        for (int ks = 0; ks < ksteps; ++ks) {
          const uint64_t da = sm100::umma_desc_sw128(st + (ks >> 2) * kBlock) + (ks & 3) * 2;
          const uint64_t db = sm100::umma_desc_sw128(q_s + (ks >> 2) * N * 128) + (ks & 3) * 2;
          sm100::umma_bf16(d, da, db, idesc_s, ks > 0 ? 1u : 0u);
        }
        sm100::umma_commit(&bars.s_full[t & 1]);
      };
      auto issue_pv = [&](int t) {
        const uint32_t st = base + (t % stages) * stage_bytes;
        for (int m = 0; m < mblocks; ++m) {
          const uint32_t d = tmem + kOCol + static_cast<uint32_t>(m * N);
#pragma unroll
          for (int kk = 0; kk < kTile / 16; ++kk) {
            const uint64_t da = sm100::umma_desc_mn_sw128(st + m * 2 * kBlock + kk * 2048, kBlock, 1024);
            sm100::umma_bf16(d, da, sm100::umma_desc_sw128(p_s) + kk * 2, idesc_o, (t > 0 || kk > 0) ? 1u : 0u);
            sm100::umma_bf16(d, da, sm100::umma_desc_sw128(p_s + N * 128) + kk * 2, idesc_o, 1u);
          }
        }
        sm100::umma_commit(&bars.pv_done);
        sm100::umma_commit(&bars.kv_empty[t % stages]);
      };
      bool ok = wait_bar(&bars.q_full, 0, &bars, 2) && wait_bar(&bars.kv_full[0], 0, &bars, 3);
      if (ok) {
        sm100::tc_fence_after_sync();
        issue_s(0);
      }
      for (int t = 0; ok && t < tiles; ++t) {
        if (t + 1 < tiles) {
          ok = wait_bar(&bars.kv_full[(t + 1) % stages], ((t + 1) / stages) & 1, &bars, 4);
          if (ok) {
            // S^T(t - 1), which the buffer held, was read before p_full(t - 1)
            sm100::tc_fence_after_sync();
            issue_s(t + 1);
          }
        }
        if (ok) ok = wait_bar(&bars.p_full, t & 1, &bars, 5);
        if (ok) {
          sm100::tc_fence_after_sync();
          issue_pv(t);
        }
      }
    }
    __syncwarp();
  } else if (warp < 4) {
    // ------------------------------------------------------------------ softmax, epilogue
    const uint32_t lane_off = static_cast<uint32_t>(warp * 32) << 16;
    const float qscale = a.scale * kLog2e;
    float m_run[kHeads], l_run[kHeads];
#pragma unroll
    for (int r = 0; r < kHeads; ++r) m_run[r] = -CUDART_INF_F, l_run[r] = 0.f;
    bool ok = true;
    for (int t = 0; t < tiles; ++t) {
      ok = wait_bar(&bars.s_full[t & 1], (t >> 1) & 1, &bars, 6);
      ok = __all_sync(0xffffffffu, ok);
      if (ok && warp < 2) {
        sm100::tc_fence_after_sync();
        uint32_t sv[32];
        tmem_ld_n<N>(tmem + lane_off + static_cast<uint32_t>((t & 1) * N), sv);
        sm100::tc_fence_before_sync();
        const int tok = warp * 32 + lane;
#pragma unroll
        for (int h = 0; h < N; ++h) s_s[h * kTile + tok] = __uint_as_float(sv[h]);
      }
      if (softmax_any(!ok)) {
        ok = false;
        break;
      }
      const int live = t1 - t0 - t * kTile;
      float v[kHeads][2], mx[kHeads];
#pragma unroll
      for (int r = 0; r < kHeads; ++r) {
        const float2 x = *reinterpret_cast<const float2*>(s_s + (warp * kHeads + r) * kTile + lane * 2);
        v[r][0] = lane * 2 < live ? x.x * qscale : -CUDART_INF_F;
        v[r][1] = lane * 2 + 1 < live ? x.y * qscale : -CUDART_INF_F;
        mx[r] = fmaxf(v[r][0], v[r][1]);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int r = 0; r < kHeads; ++r) mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], o));
      float sum[kHeads];
      uint32_t hi[kHeads], lo[kHeads];
      bool rescale = false;
#pragma unroll
      for (int r = 0; r < kHeads; ++r) {
        float f = 1.f;
        if (mx[r] > m_run[r] + kRescaleStep || m_run[r] == -CUDART_INF_F) {
          if (m_run[r] != -CUDART_INF_F) {
            f = exp2f(m_run[r] - mx[r]);
            rescale = true;
          }
          m_run[r] = mx[r];
        }
        const float p0 = exp2f(v[r][0] - m_run[r]), p1 = exp2f(v[r][1] - m_run[r]);
        sum[r] = p0 + p1;
        l_run[r] *= f;
        const __nv_bfloat162 h2 = __floats2bfloat162_rn(p0, p1);
        const float2 hf = __bfloat1622float2(h2);
        const __nv_bfloat162 l2 = __floats2bfloat162_rn(p0 - hf.x, p1 - hf.y);
        hi[r] = *reinterpret_cast<const uint32_t*>(&h2);
        lo[r] = *reinterpret_cast<const uint32_t*>(&l2);
        if (lane == 0) f_s[warp * kHeads + r] = f;
      }
      if (lane == 0) r_s[warp] = rescale ? 1u : 0u;   // the decision is the same in every lane
      // the second product of the tile before reads P^T and adds to O^T until here
      if (t > 0) ok = __all_sync(0xffffffffu, wait_bar(&bars.pv_done, (t - 1) & 1, &bars, 7));
#pragma unroll
      for (int r = 0; r < kHeads; ++r) {
        const int h = warp * kHeads + r;
        // 16-byte pieces of a head's 128-byte row, XOR-swizzled by the row like a TMA-written tile
        const uint32_t off = static_cast<uint32_t>(h * 128 + (((lane >> 2) ^ (h & 7)) << 4) + (lane & 3) * 4);
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(p_s + off), "r"(hi[r]) : "memory");
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(p_s + N * 128 + off), "r"(lo[r]) : "memory");
      }
      if (live < kTile) {
        // cache rows past the sequence may hold anything: their probability is zero, their values must be too
        const uint32_t st = base + (t % stages) * stage_bytes;
        const int per = (kTile - live) * 8;             // 16-byte pieces per block
        for (int i = threadIdx.x; i < per * blocks; i += 128) {
          const uint32_t p = st + (i / per) * kBlock + live * 128 + (i % per) * 16;
          asm volatile("st.shared.v4.u32 [%0], {%1, %1, %1, %1};" ::"r"(p), "r"(0u) : "memory");
        }
      }
      sm100::fence_proxy_async_smem();                // this thread's stores, for the tensor core's reads
      if (softmax_any(!ok)) {
        ok = false;
        break;
      }
      if ((r_s[0] | r_s[1] | r_s[2] | r_s[3]) != 0) {
        sm100::tc_fence_after_sync();
        for (int m = 0; m < mblocks; ++m) {
          const uint32_t addr = tmem + lane_off + kOCol + static_cast<uint32_t>(m * N);
#pragma unroll
          for (int c = 0; c < N; c += 16) {
            float o[16];
            sm100::tmem_ld16(addr + c, o);
            uint32_t w[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) w[j] = __float_as_uint(o[j] * f_s[c + j]);
            sm100::tmem_st16(addr + c, w);
          }
        }
        sm100::tmem_st_wait();
      }
      sm100::tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) sm100::mbar_arrive(&bars.p_full);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int r = 0; r < kHeads; ++r) sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], o);
#pragma unroll
      for (int r = 0; r < kHeads; ++r) l_run[r] += sum[r];
    }
    if (ok && tiles > 0) ok = __all_sync(0xffffffffu, wait_bar(&bars.pv_done, (tiles - 1) & 1, &bars, 8));
    if (lane == 0) {
#pragma unroll
      for (int r = 0; r < kHeads; ++r) {
        const int h = warp * kHeads + r;
        m_s[h] = m_run[r];
        l_s[h] = l_run[r];
      }
    }
    if (!softmax_any(!ok)) {
      // head h's factor: 1 / sum and the gate (a slice of a split row leaves both to the merge)
      if (threadIdx.x < N) {
        const int h = threadIdx.x;
        float f = 1.f;
        if (a.num_splits <= 1) {
          f = tiles > 0 ? 1.f / l_s[h] : 0.f;
          if (a.gate != nullptr && h < nh)
            f *= elem::sigmoid(elem::ld(reinterpret_cast<const __nv_bfloat16*>(a.gate) + static_cast<size_t>(row) * a.ld_gate + h0 + h));
        }
        f_s[h] = f;
      }
      softmax_any(false);
      sm100::tc_fence_after_sync();
      for (int m = 0; m < mblocks; ++m) {
        const int c = m * 128 + warp * 32 + lane;      // latent column = tensor-memory lane
        uint32_t ov[32];
#pragma unroll
        for (int h = 0; h < 32; ++h) ov[h] = 0u;
        if (tiles > 0) tmem_ld_n<N>(tmem + lane_off + kOCol + static_cast<uint32_t>(m * N), ov);
        if (c < a.kv_rank) {
#pragma unroll
          for (int h = 0; h < N; ++h) {
            if (h < nh) {
              const float x = __uint_as_float(ov[h]);
              if (a.num_splits > 1)
                a.ws[((static_cast<size_t>(row) * a.heads + h0 + h) * a.num_splits + split) * (a.kv_rank + 2) + c] = x;
              else
                reinterpret_cast<__nv_bfloat16*>(a.out)[(static_cast<size_t>(h0 + h) * a.q_rows + row) * a.ld_out + c] =
                    __float2bfloat16_rn(x * f_s[h]);
            }
          }
        }
      }
      if (a.num_splits > 1 && static_cast<int>(threadIdx.x) < nh) {
        float* w = a.ws + ((static_cast<size_t>(row) * a.heads + h0 + threadIdx.x) * a.num_splits + split) * (a.kv_rank + 2);
        w[a.kv_rank] = m_s[threadIdx.x];
        w[a.kv_rank + 1] = l_s[threadIdx.x];
      }
    }
  }
  // -------------------------------------------------------------------- common exit
  sm100::tc_fence_before_sync();
  __syncthreads();
  if (bars.abort_flag != 0) {
    if (threadIdx.x == 0 && a.status != nullptr && atomicCAS(a.status, 0u, 8u) == 0u) {
      a.status[1] = bars.abort_flag;
      a.status[2] = (blockIdx.z << 16) | (blockIdx.y << 8) | blockIdx.x;
      a.status[3] = static_cast<uint32_t>(tiles);
    }
    __nanosleep(1000000);   // copies still in flight get a bounded chance to land before the CTA retires
  }
  if (warp == 5) {
    sm100::tc_fence_after_sync();
    sm100::tmem_dealloc(tmem, kTmemCols);
  }
}

template <int N>
static int launch(const XpLatentAttnArgs& a, cudaStream_t s) {
  const Layout L = layout(a.ld_cache, N);
  if (L.total > kMaxDynamic) return 1;
  CUtensorMap mq, mkv;
  const int box = a.page_size % kTile == 0 ? kTile : 16;
  if (tmap::cache().get(&mkv, a.cache, static_cast<uint64_t>(a.num_pages) * a.page_size, a.ld_cache, static_cast<uint64_t>(a.ld_cache) * 2,
                        box, 2) != 0)
    return -20;
  if (tmap::cache().get_heads(&mq, a.q, a.ld_q, a.q_rows, a.heads, N) != 0) return -20;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(latent_attn_umma_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynamic) != cudaSuccess) return -21;
    set = true;
  }
  dim3 grid(a.num_splits > 1 ? a.num_splits : 1, (a.heads + N - 1) / N, a.rows);
  latent_attn_umma_kernel<N><<<grid, kThreads, L.total, s>>>(mq, mkv, a, box);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -100 - static_cast<int>(e);
}

}  // namespace latent5
}  // namespace xpool

// Returns 1 when the arguments are outside what the kernel covers, 0 when it was launched (the caller merges the slices of
// a split run), a negative code on failure.
extern "C" int xp_latent_attn_umma(const XpLatentAttnArgs* a, void* stream) {
  using namespace xpool::latent5;
  const bool ok = !a->f32 && a->kv_rank <= 512 && a->num_pages > 0 && a->page_size % 16 == 0 && a->ld_cache % 16 == 0 &&
                  a->ld_q % 16 == 0 && a->ld_q >= a->ld_cache && (a->num_splits <= 1 || a->chunk_tokens % kTile == 0) &&
                  reinterpret_cast<uintptr_t>(a->q) % 16 == 0 && reinterpret_cast<uintptr_t>(a->cache) % 16 == 0;
  if (!ok) return 1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->heads > 16 ? launch<32>(*a, s) : launch<16>(*a, s);
}
