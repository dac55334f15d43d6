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
constexpr int kScan = 512;                 // threads of a scanning CTA
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
  float b[5][D];                           // running sums before each block, and behind the last
};

// log2 of sigmoid(z) ** inv_tau; the logarithm of 1 + e keeps its relative accuracy for small e
__device__ __forceinline__ float log2_decay(float z, float inv_tau) {
  const float x = -kLog2e * z, e = sm100::ex2_approx(-fabsf(x));
  float l;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(l) : "f"(1.f + e));
  if (e < 0.03125f) l = kLog2e * e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 0.33333333f), -0.5f), 1.f);
  return -(fmaxf(x, 0.f) + l) * inv_tau;
}

// A thread takes two channels of one block: 16 tokens, all loads in flight at once.
template <int D>
__global__ void __launch_bounds__(256)
gated_linear_chunk_kernel(XpGatedLinearArgs a) {
  constexpr int PD = D + 8, kPairs = D / 2;
  extern __shared__ __align__(16) uint8_t smem[];
  ChunkSmem<D>& sm = *reinterpret_cast<ChunkSmem<D>*>(smem);
  const int h = blockIdx.y, seq = blockIdx.z, total = a.q_lens[seq];
  const int t0 = blockIdx.x * kChunk;
  if (t0 >= total) return;
  const int n = min(kChunk, total - t0), r0 = a.q_starts[seq] + t0;
  const int width = a.heads * a.dim;
  float* z = const_cast<float*>(a.z) + static_cast<size_t>(r0) * width + h * a.dim;
  const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(a.proj) + static_cast<size_t>(r0) * a.ld_proj + h * a.dim;
  const int d = threadIdx.x % kPairs * 2, blk = threadIdx.x / kPairs;
  const bool mine = blk < 4;
  float2 c[16];
  uint32_t q[16], k[16];
  bool far = false;
  if (mine) {
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      const int row = blk * 16 + t;
      const bool ok = row < n && d < a.dim;
      const __nv_bfloat16* p = rows + static_cast<size_t>(ok ? row : 0) * a.ld_proj + (ok ? d : 0);
      c[t] = ok ? *reinterpret_cast<const float2*>(z + static_cast<size_t>(row) * width + d) : make_float2(0.f, 0.f);
      q[t] = ok ? *reinterpret_cast<const uint32_t*>(p + a.q_off) : 0u;
      k[t] = ok ? *reinterpret_cast<const uint32_t*>(p + a.k_off) : 0u;
    }
    float2 s = make_float2(0.f, 0.f);
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      if (blk * 16 + t < n && d < a.dim) s.x += log2_decay(c[t].x, a.inv_tau), s.y += log2_decay(c[t].y, a.inv_tau);
      c[t] = s;
    }
    *reinterpret_cast<float2*>(&sm.b[blk + 1][d]) = s;
    far = s.x < -kRange || s.y < -kRange;
  }
  const bool direct = __syncthreads_or(far) != 0;
  // the blocks' starts
  for (int i = threadIdx.x; i < D; i += 256) {
    float s = 0.f;
    sm.b[0][i] = 0.f;
#pragma unroll
    for (int r = 1; r < 5; ++r) sm.b[r][i] = s += sm.b[r][i];
  }
  __syncthreads();
  // c to the workspace; queries and keys with what their own block decays them
  if (mine) {
    const float2 start = *reinterpret_cast<const float2*>(&sm.b[blk][d]);
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      const int row = blk * 16 + t;
      if (row < n && d < a.dim) *reinterpret_cast<float2*>(z + static_cast<size_t>(row) * width + d) = make_float2(start.x + c[t].x, start.y + c[t].y);
      float2 x = unpack2(q[t]), y = unpack2(k[t]);
      x.x *= a.qscale, x.y *= a.qscale;
      if (!direct) {
        x.x *= sm100::ex2_approx(c[t].x), x.y *= sm100::ex2_approx(c[t].y);
        y.x *= sm100::ex2_approx(-c[t].x), y.y *= sm100::ex2_approx(-c[t].y);
      }
      uint32_t hi, lo;
      split2(x.x, x.y, hi, lo);
      *reinterpret_cast<uint32_t*>(sm.q[0] + row * PD + d) = hi;
      *reinterpret_cast<uint32_t*>(sm.q[1] + row * PD + d) = lo;
      split2(y.x, y.y, hi, lo);
      *reinterpret_cast<uint32_t*>(sm.k[0] + row * PD + d) = hi;
      *reinterpret_cast<uint32_t*>(sm.k[1] + row * PD + d) = lo;
    }
  }
  __syncthreads();                         // also makes c visible to the block
  Record* rec = reinterpret_cast<Record*>(a.records) + static_cast<size_t>(first_record(a.q_starts[seq], seq) + blockIdx.x) * a.heads + h;
  if (direct) {                            // q and k are undecayed here
    for (int p = threadIdx.x; p < kChunk * kChunk; p += 256) {
      const int i = p / kChunk, j = p % kChunk;
      float s = 0.f;
      if (j <= i && i < n) {
        for (int e = 0; e < a.dim; ++e) {
          const float x = z[static_cast<size_t>(i) * width + e] - z[static_cast<size_t>(j) * width + e];
          const float qe = __bfloat162float(sm.q[0][i * PD + e]) + __bfloat162float(sm.q[1][i * PD + e]);
          const float ke = __bfloat162float(sm.k[0][j * PD + e]) + __bfloat162float(sm.k[1][j * PD + e]);
          s = fmaf(qe * ke, exp2f(x), s);
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
          const int e = ks * 16 + u * 8 + q4 * 2;
          const float f0 = sm100::ex2_approx(sm.b[rw][e] - sm.b[j][e]), f1 = sm100::ex2_approx(sm.b[rw][e + 1] - sm.b[j][e + 1]);
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
__global__ void __launch_bounds__(kScan, 1)
gated_linear_scan_kernel(XpGatedLinearArgs a) {
  constexpr int PD = D + 8, PV = VS + 8;
  constexpr int NO = VS / 32 > 1 ? VS / 32 : 2;      // output tiles of a warp (8 columns each; 16 rows)
  constexpr int kOut = VS / (8 * NO);                // warps side by side there
  constexpr int NS = D >= 128 ? VS / 16 : VS / 32 > 1 ? VS / 32 : 2;   // state column tiles of a warp (16 rows)
  constexpr int kRowWarps = D / 16, kState = VS / (8 * NS);
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
      for (int i = threadIdx.x; i < kChunk * kPieces; i += kScan) {
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
      for (int i = threadIdx.x; i < kChunk * kVPieces; i += kScan) {
        const int t = i / kVPieces, e = i % kVPieces * 8;
        const bool ok = t < m && c0 + e < a.vdim;
        copy16(sm.v[b] + t * PV + e, rows + static_cast<size_t>(ok ? t : 0) * a.ld_proj + (ok ? c0 + e : 0), ok);
      }
      if (kFull) {
        const Record* rec = recs + static_cast<size_t>(c) * a.heads;
#pragma unroll
        for (int p = 0; p < 2; ++p)
#pragma unroll
          for (int i = threadIdx.x; i < kChunk * 8; i += kScan) {
            const int t = i >> 3, e = (i & 7) * 8;
            if (e / 16 <= t / 16) copy16(sm.a[b][p] + t * kPC + e, rec->a[p] + t * kChunk + e, true);   // lower blocks only
          }
      }
    }
  };
  issue_rows(0);
  issue_tiles(0);
  copies_issued();

  const int d0 = warp % kRowWarps * 16, s0 = warp / kRowWarps * (NS * 8);
  const bool has_state = warp / kRowWarps < kState;
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
      if (has_state && !zero && d < a.dim && c < a.vdim) x = make_float2(from[static_cast<size_t>(d) * a.vdim + c], from[static_cast<size_t>(d) * a.vdim + c + 1]);
      s[j][2 * r] = x.x;
      s[j][2 * r + 1] = x.y;
    }
  auto publish = [&]() {
    if (!has_state) return;
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

  const int rw = warp & 3, o0 = (warp >> 2) * (NO * 8);
  for (int c = 0; c < chunks; ++c) {
    const int b = c & 1, m = min(kChunk, n - c * kChunk);
    copies_wait<0>();
    __syncthreads();                                 // chunk c landed, state published, everything of chunk c - 1 used
    // ---- decay queries and keys
    {
      constexpr int kPairs = D / 2, kRows = kScan / kPairs;
      const int e = threadIdx.x % kPairs * 2;
      const float2 end = *reinterpret_cast<const float2*>(sm.c_in + (m - 1) * D + e);
#pragma unroll 4
      for (int t = threadIdx.x / kPairs; t < kChunk; t += kRows) {
        const float2 cc = *reinterpret_cast<const float2*>(sm.c_in + t * D + e);
        uint32_t hi, lo;
        if (kFull) {
          const float2 x = unpack2(*reinterpret_cast<const uint32_t*>(sm.q_in + t * D + e));
          split2(x.x * (a.qscale * sm100::ex2_approx(cc.x)), x.y * (a.qscale * sm100::ex2_approx(cc.y)), hi, lo);
          *reinterpret_cast<uint32_t*>(sm.q[0] + t * PD + e) = hi;
          *reinterpret_cast<uint32_t*>(sm.q[1] + t * PD + e) = lo;
        }
        const float2 x = unpack2(*reinterpret_cast<const uint32_t*>(sm.k_in + t * D + e));   // zeros behind the portion
        const bool in = t < m;
        split2(in ? x.x * sm100::ex2_approx(end.x - cc.x) : 0.f, in ? x.y * sm100::ex2_approx(end.y - cc.y) : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(sm.k[0] + t * PD + e) = hi;
        *reinterpret_cast<uint32_t*>(sm.k[1] + t * PD + e) = lo;
      }
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
      if (warp >> 2 < kOut) {
        float o[2][NO][4];                           // two chains of sums
#pragma unroll
        for (int p = 0; p < 2; ++p)
#pragma unroll
          for (int j = 0; j < NO; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[p][j][e] = 0.f;
        const uint32_t qh_a = sm100::smem_u32(sm.q[0] + rw * 16 * PD) + a_lane(lane, PD), ql_a = sm100::smem_u32(sm.q[1] + rw * 16 * PD) + a_lane(lane, PD);
        const uint32_t sh = sm100::smem_u32(sm.s[0] + o0) + bt_lane(lane, PV), sl = sm100::smem_u32(sm.s[1] + o0) + bt_lane(lane, PV);
#pragma unroll 4
        for (int ks = 0; ks < D / 16; ++ks) {
          uint32_t qh[4], ql[4];
          ldsm4(qh_a + ks * 32, qh);
          ldsm4(ql_a + ks * 32, ql);
#pragma unroll
          for (int j = 0; j < NO; j += 2) {
            uint32_t hi[4], lo[4];
            ldsm4t(sh + (ks * 16 * PV + j * 8) * 2, hi);
            ldsm4t(sl + (ks * 16 * PV + j * 8) * 2, lo);
            mma(o[0][j], qh, hi[0], hi[1]);
            mma(o[0][j + 1], qh, hi[2], hi[3]);
            mma(o[1][j], qh, lo[0], lo[1]);
            mma(o[1][j + 1], qh, lo[2], lo[3]);
            mma(o[1][j], ql, hi[0], hi[1]);
            mma(o[1][j + 1], ql, hi[2], hi[3]);
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
              mma(o[0][j], ah, vf[0], vf[1]);
              mma(o[0][j + 1], ah, vf[2], vf[3]);
              mma(o[1][j], al, vf[0], vf[1]);
              mma(o[1][j + 1], al, vf[2], vf[3]);
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
                  make_float2(o[0][j][2 * r] + o[1][j][2 * r], o[0][j][2 * r + 1] + o[1][j][2 * r + 1]);
          }
        }
      }
      if (c + 1 == chunks && !last) break;           // the next segment has its own start state
      __syncthreads();                               // everyone is done with the published state
    }
    if (has_state) {
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
      if (has_state && d < a.dim && c < a.vdim) {
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
    gated_linear_scan_kernel<D, VS, false><<<grid, kScan, kScanBytes, s>>>(b);
    gated_linear_segments_kernel<<<dim3((a.dim * a.vdim + 255) / 256, a.heads, a.seqs), 256, 0, s>>>(b);
  }
  gated_linear_scan_kernel<D, VS, true><<<grid, kScan, kScanBytes, s>>>(b);
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
