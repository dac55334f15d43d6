// Linear attention with a decay per key channel over portions of prompts, in chunks of 64 tokens on the tensor cores (bf16
// rows, up to 128 key dimensions). With c_i [dim] the running sum of log2 alpha in a chunk and S the state before it:
//   o_i = S^T (2^c_i q_i) + sum_{j <= i} A_ij v_j,    A_ij = sum_d q_id k_jd 2^(c_id - c_jd)
//   S  <- 2^c_n S + sum_j (2^(c_n - c_j) k_j) v_j^T
//   gated_linear_chunk_kernel   per (chunk, head), all at once: turns z into c in place and computes A
//   gated_linear_scan_kernel    per (segment, VS value columns, head, sequence): walks its chunks, state in registers
// A splits at blocks of 16 tokens: with b_r = c before block r, queries enter as 2^(c_i - b_r) q_i (at most q), keys as
// 2^(b_r' - c_j) k_j with their own block's b (at least k), and 2^(b_r - b_r') stands between two blocks. Where a block decays
// by more than 2^kRange in some channel, the chunk's A is summed up term by term instead.
// Decayed queries and keys, A and the state enter products as bf16 pairs (high and low part); sums are fp32.
// Long portions with few heads are cut into segments that run at the same time, as in linear_attn.cu.
#include "xpool/mixer_api.h"
#include "xpool/mma_sync.cuh"
#include "xpool/recurrence.cuh"

namespace xpool {
namespace gla {

using namespace xpool::frag;

constexpr int kChunk = 64;
constexpr int kPC = kChunk + 8;
constexpr float kRange = 80.f;
constexpr float kLog2e = 1.4426950408889634f;

struct __align__(16) Record {              // A of a (chunk, head): high parts, low parts
  __nv_bfloat16 a[2][kChunk * kChunk];
};

__device__ __forceinline__ int first_record(int start, int seq) { return start / kChunk + seq; }

template <int D>
struct ChunkSmem {
  static constexpr int PD = D + 8;
  __nv_bfloat16 q[2][kChunk * PD], k[2][kChunk * PD];
  float c[kChunk * D];                     // running sums
  float b[4][D];                           // ... before each block
};

template <int D>
__global__ void __launch_bounds__(256)
gated_linear_chunk_kernel(XpGatedLinearArgs a) {
  constexpr int PD = D + 8;
  extern __shared__ __align__(16) uint8_t smem[];
  ChunkSmem<D>& sm = *reinterpret_cast<ChunkSmem<D>*>(smem);
  __shared__ int wide;
  const int h = blockIdx.y, seq = blockIdx.z, total = a.q_lens[seq];
  const int t0 = blockIdx.x * kChunk;
  if (t0 >= total) return;
  const int n = min(kChunk, total - t0), r0 = a.q_starts[seq] + t0;
  const int width = a.heads * a.dim;
  float* z = const_cast<float*>(a.z) + static_cast<size_t>(r0) * width + h * a.dim;
  const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(a.proj) + static_cast<size_t>(r0) * a.ld_proj + h * a.dim;
  if (threadIdx.x == 0) wide = 0;
  for (int i = threadIdx.x; i < kChunk * D; i += 256) {
    const int t = i / D, d = i % D;
    sm.c[i] = t < n && d < a.dim ? recur::log_decay(z[static_cast<size_t>(t) * width + d], a.inv_tau) * kLog2e : 0.f;
  }
  __syncthreads();
  // sums inside each block of 16 tokens, then the blocks' starts
  for (int i = threadIdx.x; i < 4 * D; i += 256) {
    const int d = i % D, r = i / D;
    float s = 0.f;
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      s += sm.c[(r * 16 + t) * D + d];
      sm.c[(r * 16 + t) * D + d] = s;
    }
    if (s < -kRange) wide = 1;
  }
  __syncthreads();
  for (int d = threadIdx.x; d < D; d += 256) {
    float s = 0.f;
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      sm.b[r][d] = s;
      s += sm.c[(r * 16 + 15) * D + d];
    }
  }
  __syncthreads();
  // c to the workspace; decayed queries and keys (of both only what their own block adds)
  const bool direct = wide != 0;
  constexpr int kPieces = D / 8;
  for (int i = threadIdx.x; i < kChunk * kPieces; i += 256) {
    const int t = i / kPieces, e = i % kPieces * 8, r = t >> 4;
    const bool ok = t < n && e < a.dim;
    float q[8], k[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) q[j] = k[j] = 0.f;
    if (ok) {
      recur::ldx<8>(rows + static_cast<size_t>(t) * a.ld_proj + a.q_off + e, q);
      recur::ldx<8>(rows + static_cast<size_t>(t) * a.ld_proj + a.k_off + e, k);
    }
    float4 c[2];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float x = sm.c[t * D + e + j];
      reinterpret_cast<float*>(c)[j] = x + sm.b[r][e + j];
      q[j] *= a.qscale;
      if (!direct) {
        q[j] *= sm100::ex2_approx(x);
        k[j] *= sm100::ex2_approx(-x);
      }
    }
    if (ok) {
      *reinterpret_cast<float4*>(z + static_cast<size_t>(t) * width + e) = c[0];
      *reinterpret_cast<float4*>(z + static_cast<size_t>(t) * width + e + 4) = c[1];
    }
    uint4 hi, lo;
    split2(q[0], q[1], hi.x, lo.x), split2(q[2], q[3], hi.y, lo.y), split2(q[4], q[5], hi.z, lo.z), split2(q[6], q[7], hi.w, lo.w);
    *reinterpret_cast<uint4*>(sm.q[0] + t * PD + e) = hi;
    *reinterpret_cast<uint4*>(sm.q[1] + t * PD + e) = lo;
    split2(k[0], k[1], hi.x, lo.x), split2(k[2], k[3], hi.y, lo.y), split2(k[4], k[5], hi.z, lo.z), split2(k[6], k[7], hi.w, lo.w);
    *reinterpret_cast<uint4*>(sm.k[0] + t * PD + e) = hi;
    *reinterpret_cast<uint4*>(sm.k[1] + t * PD + e) = lo;
  }
  __syncthreads();
  Record* rec = reinterpret_cast<Record*>(a.records) + static_cast<size_t>(first_record(a.q_starts[seq], seq) + blockIdx.x) * a.heads + h;
  if (direct) {                            // q and k are undecayed here
    for (int p = threadIdx.x; p < kChunk * kChunk; p += 256) {
      const int i = p / kChunk, j = p % kChunk;
      float s = 0.f;
      if (j <= i) {
        for (int d = 0; d < a.dim; ++d) {
          const float x = (sm.c[i * D + d] - sm.c[j * D + d]) + (sm.b[i >> 4][d] - sm.b[j >> 4][d]);
          const float q = __bfloat162float(sm.q[0][i * PD + d]) + __bfloat162float(sm.q[1][i * PD + d]);
          const float k = __bfloat162float(sm.k[0][j * PD + d]) + __bfloat162float(sm.k[1][j * PD + d]);
          s = fmaf(q * k, exp2f(x), s);
        }
      }
      const __nv_bfloat16 hi = __float2bfloat16_rn(s);
      rec->a[0][p] = hi;
      rec->a[1][p] = __float2bfloat16_rn(s - __bfloat162float(hi));
    }
    return;
  }
  // warp: 16 rows, half of the key blocks (0 and 2, or 1 and 3)
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q4 = lane & 3, rw = warp & 3, half = warp >> 2;
  const uint32_t qa_hi = sm100::smem_u32(sm.q[0] + rw * 16 * PD) + a_lane(lane, PD), qa_lo = sm100::smem_u32(sm.q[1] + rw * 16 * PD) + a_lane(lane, PD);
  const uint32_t kb_hi = sm100::smem_u32(sm.k[0]) + b_lane(lane, PD), kb_lo = sm100::smem_u32(sm.k[1]) + b_lane(lane, PD);
#pragma unroll
  for (int jj = 0; jj < 2; ++jj) {
    const int j = jj * 2 + half;
    if (j > rw) break;
    float p[2][4];
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int e = 0; e < 4; ++e) p[u][e] = 0.f;
#pragma unroll 2
    for (int ks = 0; ks < D / 16; ++ks) {
      uint32_t qh[4], ql[4], kh[4], kl[4];
      ldsm4(qa_hi + ks * 32, qh);
      ldsm4(qa_lo + ks * 32, ql);
      ldsm4(kb_hi + (j * 16 * PD + ks * 16) * 2, kh);
      ldsm4(kb_lo + (j * 16 * PD + ks * 16) * 2, kl);
      if (j < rw) {                        // what lies between the two blocks
#pragma unroll
        for (int u = 0; u < 2; ++u) {      // dims d, d + 1 and d + 8, d + 9 of the fragment
          const int d = ks * 16 + u * 8 + q4 * 2;
          const float f0 = sm100::ex2_approx(sm.b[rw][d] - sm.b[j][d]), f1 = sm100::ex2_approx(sm.b[rw][d + 1] - sm.b[j][d + 1]);
#pragma unroll
          for (int v = 0; v < 2; ++v) {    // rows g and g + 8
            const float2 x = unpack2(qh[u * 2 + v]), y = unpack2(ql[u * 2 + v]);
            split2((x.x + y.x) * f0, (x.y + y.y) * f1, qh[u * 2 + v], ql[u * 2 + v]);
          }
        }
      }
      mma(p[0], qh, kh[0], kh[1]);
      mma(p[1], qh, kh[2], kh[3]);
      mma(p[0], qh, kl[0], kl[1]);
      mma(p[1], qh, kl[2], kl[3]);
      mma(p[0], ql, kh[0], kh[1]);
      mma(p[1], ql, kh[2], kh[3]);
    }
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int i = rw * 16 + g + r * 8, at = j * 16 + u * 8 + q4 * 2;
        uint32_t hi, lo;
        split2(at <= i ? p[u][2 * r] : 0.f, at + 1 <= i ? p[u][2 * r + 1] : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(rec->a[0] + i * kChunk + at) = hi;
        *reinterpret_cast<uint32_t*>(rec->a[1] + i * kChunk + at) = lo;
      }
  }
}

template <int D, int VS>
struct ScanSmem {
  static constexpr int PD = D + 8, PV = VS + 8;
  __nv_bfloat16 q_in[kChunk * D], k_in[kChunk * D];  // rows as they come
  float c_in[kChunk * D];
  __nv_bfloat16 v[2][kChunk * PV];
  __nv_bfloat16 a[2][2][kChunk * kPC];
  __nv_bfloat16 q[2][kChunk * PD], k[2][kChunk * PD];   // decayed, high and low parts
  __nv_bfloat16 s[2][D * PV];              // state
  float dec[D];                            // 2^c_n
};

// kFull: outputs and the state; otherwise only what the segment adds to the state, and its decay.
template <int D, int VS, bool kFull>
__global__ void __launch_bounds__(256, 1)
gated_linear_scan_kernel(XpGatedLinearArgs a) {
  constexpr int PD = D + 8, PV = VS + 8;
  constexpr int NO = VS / 16;                        // output tiles of a warp (half of the columns, 8 each)
  constexpr int NS = D >= 128 ? VS / 8 : VS / 16;    // state column tiles of a warp
  extern __shared__ __align__(16) uint8_t smem[];
  ScanSmem<D, VS>& sm = *reinterpret_cast<ScanSmem<D, VS>*>(smem);
  const int slices = (a.vdim + VS - 1) / VS;
  const int seg = blockIdx.x / slices, c0 = (blockIdx.x % slices) * VS;
  const int h = blockIdx.y, seq = blockIdx.z, total = a.q_lens[seq];
  const int first = seg * a.seg_tokens;              // segments are whole chunks long
  if (first >= total) return;
  const bool last = first + a.seg_tokens >= total;
  if (!kFull && last) return;                        // nobody starts behind the last segment
  const int n = min(a.seg_tokens, total - first), r0 = a.q_starts[seq] + first;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q4 = lane & 3;
  const int chunks = (n + kChunk - 1) / kChunk, width = a.heads * a.dim;
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(a.proj);
  const Record* recs = reinterpret_cast<const Record*>(a.records) + static_cast<size_t>(first_record(a.q_starts[seq], seq) + first / kChunk) * a.heads + h;

  auto issue_rows = [&](int c) {                     // single buffers, free once the chunk before is decayed
    if (c < chunks) {
      const int m = min(kChunk, n - c * kChunk);
      const __nv_bfloat16* rows = proj + static_cast<size_t>(r0 + c * kChunk) * a.ld_proj + h * a.dim;
      const float* cs = a.z + static_cast<size_t>(r0 + c * kChunk) * width + h * a.dim;
      constexpr int kPieces = D / 8;
#pragma unroll
      for (int i = threadIdx.x; i < kChunk * kPieces; i += 256) {
        const int t = i / kPieces, e = i % kPieces * 8;
        const bool ok = t < m && e < a.dim;
        const __nv_bfloat16* row = rows + static_cast<size_t>(ok ? t : 0) * a.ld_proj + (ok ? e : 0);
        if (kFull) copy16(sm.q_in + t * D + e, row + a.q_off, ok);
        copy16(sm.k_in + t * D + e, row + a.k_off, ok);
        const float* crow = cs + static_cast<size_t>(ok ? t : 0) * width + (ok ? e : 0);
        copy16(sm.c_in + t * D + e, crow, ok);
        copy16(sm.c_in + t * D + e + 4, crow + 4, ok);
      }
    }
  };
  auto issue_tiles = [&](int c) {                    // two buffers
    if (c < chunks) {
      const int b = c & 1, m = min(kChunk, n - c * kChunk);
      const __nv_bfloat16* rows = proj + static_cast<size_t>(r0 + c * kChunk) * a.ld_proj + a.v_off + h * a.vdim;
      constexpr int kVPieces = VS / 8;
#pragma unroll
      for (int i = threadIdx.x; i < kChunk * kVPieces; i += 256) {
        const int t = i / kVPieces, e = i % kVPieces * 8;
        const bool ok = t < m && c0 + e < a.vdim;
        copy16(sm.v[b] + t * PV + e, rows + static_cast<size_t>(ok ? t : 0) * a.ld_proj + (ok ? c0 + e : 0), ok);
      }
      if (kFull) {
        const Record* rec = recs + static_cast<size_t>(c) * a.heads;
#pragma unroll
        for (int p = 0; p < 2; ++p)
#pragma unroll
          for (int i = threadIdx.x; i < kChunk * 8; i += 256) {
            const int t = i >> 3, e = (i & 7) * 8;
            if (e / 16 <= t / 16) copy16(sm.a[b][p] + t * kPC + e, rec->a[p] + t * kChunk + e, true);   // lower blocks only
          }
      }
    }
  };
  issue_rows(0);
  issue_tiles(0);
  copies_issued();

  const int d0 = D >= 128 ? warp * 16 : (warp & 3) * 16, s0 = D >= 128 ? 0 : (warp >> 2) * (VS / 2);
  const size_t state_elems = static_cast<size_t>(a.dim) * a.vdim;
  float* slot = a.state + (static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * state_elems;
  // segments: state before (or what is added) [dim][vdim], then log2 of the decay [dim]
  float* mid = a.ws + ((static_cast<size_t>(seq) * a.heads + h) * a.segs + seg) * (state_elems + a.dim);
  const float* from = kFull && a.segs > 1 ? mid : slot;
  const bool zero = !kFull || (a.segs == 1 && a.positions[r0] == 0);
  float s[NS][4];
#pragma unroll
  for (int j = 0; j < NS; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + g + r * 8, c = c0 + s0 + j * 8 + q4 * 2;
      float2 x = make_float2(0.f, 0.f);
      if (!zero && d < a.dim && c < a.vdim) x = make_float2(from[static_cast<size_t>(d) * a.vdim + c], from[static_cast<size_t>(d) * a.vdim + c + 1]);
      s[j][2 * r] = x.x;
      s[j][2 * r + 1] = x.y;
    }
  auto publish = [&]() {
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        uint32_t hi, lo;
        split2(s[j][2 * r], s[j][2 * r + 1], hi, lo);
        const int at = (d0 + g + r * 8) * PV + s0 + j * 8 + q4 * 2;
        *reinterpret_cast<uint32_t*>(sm.s[0] + at) = hi;
        *reinterpret_cast<uint32_t*>(sm.s[1] + at) = lo;
      }
  };
  if (kFull) publish();
  float log_total = 0.f;                             // thread d: log2 of channel d's decay over the segment

  const int rw = warp & 3, o0 = (warp >> 2) * (VS / 2);
  for (int c = 0; c < chunks; ++c) {
    const int b = c & 1, m = min(kChunk, n - c * kChunk);
    copies_wait<0>();
    __syncthreads();                                 // chunk c landed, state published, everything of chunk c - 1 used
    // ---- decay queries and keys
    constexpr int kPieces = D / 8;
    for (int i = threadIdx.x; i < kChunk * kPieces; i += 256) {
      const int t = i / kPieces, e = i % kPieces * 8;
      float x[8];
      uint4 hi, lo;
      float cc[8];
      *reinterpret_cast<float4*>(cc) = *reinterpret_cast<const float4*>(sm.c_in + t * D + e);
      *reinterpret_cast<float4*>(cc + 4) = *reinterpret_cast<const float4*>(sm.c_in + t * D + e + 4);
      if (kFull) {
        recur::ldx<8>(sm.q_in + t * D + e, x);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] *= a.qscale * sm100::ex2_approx(cc[j]);
        split2(x[0], x[1], hi.x, lo.x), split2(x[2], x[3], hi.y, lo.y), split2(x[4], x[5], hi.z, lo.z), split2(x[6], x[7], hi.w, lo.w);
        *reinterpret_cast<uint4*>(sm.q[0] + t * PD + e) = hi;
        *reinterpret_cast<uint4*>(sm.q[1] + t * PD + e) = lo;
      }
      recur::ldx<8>(sm.k_in + t * D + e, x);         // zeros behind the portion
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] *= t < m ? sm100::ex2_approx(sm.c_in[(m - 1) * D + e + j] - cc[j]) : 0.f;
      split2(x[0], x[1], hi.x, lo.x), split2(x[2], x[3], hi.y, lo.y), split2(x[4], x[5], hi.z, lo.z), split2(x[6], x[7], hi.w, lo.w);
      *reinterpret_cast<uint4*>(sm.k[0] + t * PD + e) = hi;
      *reinterpret_cast<uint4*>(sm.k[1] + t * PD + e) = lo;
    }
    if (threadIdx.x < D) {
      const float x = sm.c_in[(m - 1) * D + threadIdx.x];
      log_total += x;
      sm.dec[threadIdx.x] = sm100::ex2_approx(x);
    }
    __syncthreads();
    issue_rows(c + 1);
    issue_tiles(c + 1);
    copies_issued();
    const uint32_t vb = sm100::smem_u32(sm.v[b]) + bt_lane(lane, PV);
    if constexpr (kFull) {
      float o[NO][4];
#pragma unroll
      for (int j = 0; j < NO; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
      const uint32_t qh_a = sm100::smem_u32(sm.q[0] + rw * 16 * PD) + a_lane(lane, PD), ql_a = sm100::smem_u32(sm.q[1] + rw * 16 * PD) + a_lane(lane, PD);
      const uint32_t sh = sm100::smem_u32(sm.s[0] + o0) + bt_lane(lane, PV), sl = sm100::smem_u32(sm.s[1] + o0) + bt_lane(lane, PV);
#pragma unroll 2
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t qh[4], ql[4];
        ldsm4(qh_a + ks * 32, qh);
        ldsm4(ql_a + ks * 32, ql);
#pragma unroll
        for (int j = 0; j < NO; j += 2) {
          uint32_t hi[4], lo[4];
          ldsm4t(sh + (ks * 16 * PV + j * 8) * 2, hi);
          ldsm4t(sl + (ks * 16 * PV + j * 8) * 2, lo);
          mma(o[j], qh, hi[0], hi[1]);
          mma(o[j + 1], qh, hi[2], hi[3]);
          mma(o[j], qh, lo[0], lo[1]);
          mma(o[j + 1], qh, lo[2], lo[3]);
          mma(o[j], ql, hi[0], hi[1]);
          mma(o[j + 1], ql, hi[2], hi[3]);
        }
      }
      const uint32_t ah_a = sm100::smem_u32(sm.a[b][0] + rw * 16 * kPC) + a_lane(lane, kPC), al_a = sm100::smem_u32(sm.a[b][1] + rw * 16 * kPC) + a_lane(lane, kPC);
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks <= rw) {
          uint32_t ah[4], al[4];
          ldsm4(ah_a + ks * 32, ah);
          ldsm4(al_a + ks * 32, al);
#pragma unroll
          for (int j = 0; j < NO; j += 2) {
            uint32_t vf[4];
            ldsm4t(vb + (ks * 16 * PV + o0 + j * 8) * 2, vf);
            mma(o[j], ah, vf[0], vf[1]);
            mma(o[j + 1], ah, vf[2], vf[3]);
            mma(o[j], al, vf[0], vf[1]);
            mma(o[j + 1], al, vf[2], vf[3]);
          }
        }
      }
#pragma unroll
      for (int j = 0; j < NO; ++j) {
        const int col = c0 + o0 + j * 8 + q4 * 2;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int i = rw * 16 + g + r * 8;
          if (i < m && col < a.vdim)
            *reinterpret_cast<float2*>(reinterpret_cast<float*>(a.out) + static_cast<size_t>(r0 + c * kChunk + i) * a.ld_out + h * a.vdim + col) =
                make_float2(o[j][2 * r], o[j][2 * r + 1]);
        }
      }
      if (c + 1 == chunks && !last) break;           // the next segment has its own start state
      __syncthreads();                               // everyone is done with the published state
    }
    const float e0 = sm.dec[d0 + g], e1 = sm.dec[d0 + g + 8];
#pragma unroll
    for (int j = 0; j < NS; ++j) s[j][0] *= e0, s[j][1] *= e0, s[j][2] *= e1, s[j][3] *= e1;
    const uint32_t kh_a = sm100::smem_u32(sm.k[0] + d0) + at_lane(lane, PD), kl_a = sm100::smem_u32(sm.k[1] + d0) + at_lane(lane, PD);
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t kh[4], kl[4];
      ldsm4t(kh_a + ks * 16 * PD * 2, kh);
      ldsm4t(kl_a + ks * 16 * PD * 2, kl);
#pragma unroll
      for (int j = 0; j < NS; j += 2) {
        uint32_t vf[4];
        ldsm4t(vb + (ks * 16 * PV + s0 + j * 8) * 2, vf);
        mma(s[j], kh, vf[0], vf[1]);
        mma(s[j + 1], kh, vf[2], vf[3]);
        mma(s[j], kl, vf[0], vf[1]);
        mma(s[j + 1], kl, vf[2], vf[3]);
      }
    }
    if (kFull && c + 1 < chunks) publish();
  }
  copies_wait<0>();
  if (kFull && !last) return;
  float* to = kFull ? slot : mid;
#pragma unroll
  for (int j = 0; j < NS; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + g + r * 8, c = c0 + s0 + j * 8 + q4 * 2;
      if (d < a.dim && c < a.vdim) {
        to[static_cast<size_t>(d) * a.vdim + c] = s[j][2 * r];
        to[static_cast<size_t>(d) * a.vdim + c + 1] = s[j][2 * r + 1];
      }
    }
  if (!kFull && c0 == 0 && threadIdx.x < a.dim) mid[state_elems + threadIdx.x] = log_total;
}

// What each segment adds and its decay -> the state before each segment, in place.
__global__ void __launch_bounds__(256)
gated_linear_segments_kernel(XpGatedLinearArgs a) {
  const int h = blockIdx.y, seq = blockIdx.z, total = a.q_lens[seq];
  if (total <= 0) return;
  const size_t state_elems = static_cast<size_t>(a.dim) * a.vdim, pitch = state_elems + a.dim;
  const size_t i = blockIdx.x * 256ull + threadIdx.x;
  if (i >= state_elems) return;
  float* mid = a.ws + (static_cast<size_t>(seq) * a.heads + h) * a.segs * pitch;
  float x = a.positions[a.q_starts[seq]] == 0 ? 0.f : a.state[(static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * state_elems + i];
  for (int s = 0; s * a.seg_tokens < total; ++s) {
    const bool ends = (s + 1) * a.seg_tokens >= total;        // the last segment adds to nobody
    const float add = ends ? 0.f : mid[s * pitch + i], f = ends ? 0.f : exp2f(mid[s * pitch + state_elems + i / a.vdim]);
    mid[s * pitch + i] = x;
    x = fmaf(f, x, add);
  }
}

template <int D, int VS>
int launch(const XpGatedLinearArgs& a, cudaStream_t s) {
  constexpr int kChunkBytes = sizeof(ChunkSmem<D>), kScanBytes = sizeof(ScanSmem<D, VS>);
  static_assert(kScanBytes <= 227 * 1024 && kChunkBytes <= 227 * 1024, "tiles exceed the shared memory of an SM");
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(gated_linear_chunk_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, kChunkBytes) != cudaSuccess ||
        cudaFuncSetAttribute(gated_linear_scan_kernel<D, VS, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kScanBytes) != cudaSuccess ||
        cudaFuncSetAttribute(gated_linear_scan_kernel<D, VS, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kScanBytes) != cudaSuccess)
      return -21;
    attr_set = true;
  }
  XpGatedLinearArgs b = a;
  if (b.segs <= 1) {
    b.segs = 1;
    b.seg_tokens = 0x40000000;
  } else if (b.ws == nullptr || b.seg_tokens <= 0 || b.seg_tokens % kChunk != 0) {
    return -13;
  }
  gated_linear_chunk_kernel<D><<<dim3((a.max_q + kChunk - 1) / kChunk, a.heads, a.seqs), 256, kChunkBytes, s>>>(b);
  const dim3 grid((a.vdim + VS - 1) / VS * b.segs, a.heads, a.seqs);
  if (b.segs > 1) {
    gated_linear_scan_kernel<D, VS, false><<<grid, 256, kScanBytes, s>>>(b);
    gated_linear_segments_kernel<<<dim3((a.dim * a.vdim + 255) / 256, a.heads, a.seqs), 256, 0, s>>>(b);
  }
  gated_linear_scan_kernel<D, VS, true><<<grid, 256, kScanBytes, s>>>(b);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -100 - static_cast<int>(e);
}

}  // namespace gla
}  // namespace xpool

// Bytes of chunk records for batches of at most `rows` rows in `seqs` portions.
extern "C" size_t xp_gated_linear_record_bytes(int rows, int seqs, int heads) {
  return (static_cast<size_t>(rows) / xpool::gla::kChunk + seqs + 1) * heads * sizeof(xpool::gla::Record);
}

// Returns 1 when the sizes are outside what the chunked kernels cover, 0 when they were launched.
extern "C" int xp_gated_linear_chunked(const XpGatedLinearArgs* a, void* stream) {
  using namespace xpool::gla;
  const bool ok = !a->f32 && a->records != nullptr && a->max_q > 0 && a->dim <= 128 && a->dim % 8 == 0 && a->vdim % 8 == 0 && a->ld_out % 2 == 0 &&
                  a->ld_proj % 8 == 0 && a->q_off % 8 == 0 && a->k_off % 8 == 0 && a->v_off % 8 == 0 &&
                  reinterpret_cast<uintptr_t>(a->proj) % 16 == 0 && reinterpret_cast<uintptr_t>(a->records) % 16 == 0 &&
                  reinterpret_cast<uintptr_t>(a->z) % 16 == 0 && reinterpret_cast<uintptr_t>(a->out) % 8 == 0;
  if (!ok) return 1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dim <= 64) return a->vdim <= 32 ? launch<64, 32>(*a, s) : launch<64, 64>(*a, s);
  return a->vdim <= 32 ? launch<128, 32>(*a, s) : launch<128, 64>(*a, s);
}
