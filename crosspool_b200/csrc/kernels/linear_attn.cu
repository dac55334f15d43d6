// Decayed linear attention with a recurrent state per sequence and head: S <- decay S + k v^T, o = S^T q (the projection's
// epilogue has put q, k and v through silu). The state is fp32 and lives in the sequence's slot, [dim][vdim] per head; a sequence whose first
// row sits at position 0 starts from zero, so slots are handed out without clearing them.
//   linear_decode      one token per sequence: bound by reading and writing the state once
//   linear_chunked     prefill in chunks of 64 tokens on the tensor cores, bf16 inputs
//   linear_sequential  prefill as a loop over tokens, any sizes, fp32 or bf16 inputs
#include "xpool/elem.cuh"
#include "xpool/mixer_api.h"
#include "xpool/mma_sync.cuh"
#include "xpool/sm100.cuh"

namespace xpool {
namespace linear {

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
    q_s[c] = elem::ld(proj + a.q_off + h * a.dim + c);
    k_s[c] = elem::ld(proj + a.k_off + h * a.dim + c);
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
      for (int j = 0; j < N; ++j) acc[j] = 0.f;
      // kAhead rows are requested before the first of them is stored back (a store would hold back later loads)
      constexpr int kAhead = 8;
      for (int i0 = gi; i0 < a.dim; i0 += groups * kAhead) {
        float s[kAhead][N];
#pragma unroll
        for (int u = 0; u < kAhead; ++u) {
#pragma unroll
          for (int j = 0; j < N; ++j) s[u][j] = 0.f;
          if (!fresh && i0 + u * groups < a.dim) elem::ldv<N>(S + static_cast<size_t>(i0 + u * groups) * a.vdim + c, s[u]);
        }
#pragma unroll
        for (int u = 0; u < kAhead; ++u) {
          const int i = i0 + u * groups;
          if (i >= a.dim) break;
          const float ki = k_s[i], qi = q_s[i];
#pragma unroll
          for (int j = 0; j < N; ++j) {
            s[u][j] = fmaf(ki, v[j], decay * s[u][j]);
            acc[j] = fmaf(qi, s[u][j], acc[j]);
          }
          elem::stv<N>(S + static_cast<size_t>(i) * a.vdim + c, s[u]);
        }
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
  const int h = blockIdx.y, seq = blockIdx.z;
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
      q_s[i] = elem::ld(p + a.q_off);
      k_s[i] = elem::ld(p + a.k_off);
    }
    for (int i = threadIdx.x; i < m * 32; i += kThreads) {
      const int t = i >> 5, cc = blockIdx.x * 32 + (i & 31);
      v_s[i] = cc < a.vdim ? elem::ld(reinterpret_cast<const T*>(a.proj) + static_cast<size_t>(r0 + t0 + t) * a.ld_proj + a.v_off +
                                      h * a.vdim + cc)
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

// ------------------------------------------------------------------------------------------ chunked prefill
// CTA = (segment of a portion, VS state columns, head, sequence); it walks its segment in chunks of 64 tokens with the
// state in registers. With p(n) = decay^n, for row i of a chunk of n tokens and the state S before it:
//   o_i = p(i + 1) S^T q_i + sum_{j <= i} p(i - j) (q_i . k_j) v_j          (warp: 16 rows, half of the columns)
//   S   <- p(n) S + sum_j (p(n - 1 - j) k_j) v_j^T                          (warp: its 16-row tiles of S)
// Decayed scores, decayed keys and the state enter their products as bf16 pairs (high and low part), so everything
// that belongs to the recurrence keeps at least 16 mantissa bits; the sums are fp32.
//
// A long portion with few heads is cut into segments that run at the same time: a first pass computes what each segment
// adds to the state (the second line alone, from zero), a scan over the segments turns that into the state before each of
// them, and the full pass starts every segment from there.
//
// mma.sync rather than tcgen05: the state has to be scaled and re-split between chunks, which from tensor memory costs a
// round trip per chunk.
constexpr int kChunk = 64;
constexpr int kChunkThreads = 256;

using frag::ldsm4;
using frag::ldsm4t;
using frag::mma;
using frag::split2;

template <int D, int VS>
constexpr int chunk_smem_bytes() {
  // q, k [2][64][D + 8]; v [2][64][VS + 8]; state pair [2][D][VS + 8]; powers
  return (4 * kChunk * (D + 8) + 2 * kChunk * (VS + 8) + 2 * D * (VS + 8)) * 2 + (kChunk + 1 + 3) * 4;
}

// kFull: outputs and the state; otherwise only what the segment adds to the state.
template <int D, int VS, bool kFull>
__global__ void __launch_bounds__(kChunkThreads, 1)
linear_chunked_kernel(XpLinearAttnArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int PD = D + 8, PV = VS + 8;             // pitches: odd multiples of 16 bytes
  constexpr int NO = VS / 16;                        // output tiles of a warp (8 columns each)
  constexpr int MT = D > 128 ? D / 128 : 1;          // state row tiles of a warp
  constexpr int NS = D >= 128 ? VS / 8 : VS / 16;    // state column tiles of a warp
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* k_s = q_s + 2 * kChunk * PD;
  __nv_bfloat16* v_s = k_s + 2 * kChunk * PD;
  __nv_bfloat16* st_s = v_s + 2 * kChunk * PV;       // state: high parts, low parts
  float* pw = reinterpret_cast<float*>(st_s + 2 * D * PV);
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

  // columns behind dim stay zero; nothing below writes them
  if (a.dim < D) {
    const int gap = (D - a.dim) / 8;
    for (int i = threadIdx.x; i < 4 * kChunk * gap; i += kChunkThreads)
      *reinterpret_cast<uint4*>(q_s + (i / gap) * PD + a.dim + (i % gap) * 8) = make_uint4(0, 0, 0, 0);
  }
  for (int i = threadIdx.x; i <= kChunk; i += kChunkThreads) pw[i] = a.decay_pow[h * (kChunk + 1) + i];

  auto copy = [&](__nv_bfloat16* dst, const __nv_bfloat16* src, bool ok) {
    const int sz = ok ? 16 : 0;                      // rows and columns out of range read as zero
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(sm100::smem_u32(dst)), "l"(src), "r"(sz));
  };
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
          if (kFull) copy(q_s + (b * kChunk + t) * PD + e, row + a.q_off, ok);
          copy(k_s + (b * kChunk + t) * PD + e, row + a.k_off, ok);
        }
      }
      constexpr int kVPieces = VS / 8, kVRows = kChunkThreads / kVPieces;
      const int ev = (threadIdx.x % kVPieces) * 8;
#pragma unroll
      for (int t = threadIdx.x / kVPieces; t < kChunk; t += kVRows) {
        const bool ok = t < m && c0 + ev < a.vdim;
        copy(v_s + (b * kChunk + t) * PV + ev, rows + static_cast<size_t>(t < m ? t : 0) * a.ld_proj + a.v_off + h * a.vdim + (ok ? c0 + ev : 0), ok);
      }
    }
    asm volatile("cp.async.commit_group;");
  };
  issue(0);

  // the warp's part of the state
  const int d0 = D >= 128 ? warp * MT * 16 : (warp & 3) * 16;
  const int s0 = D >= 128 ? 0 : (warp >> 2) * (VS / 2);
  const size_t state_elems = static_cast<size_t>(a.dim) * a.vdim;
  float* slot = a.state + (static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * state_elems;
  float* mid = a.ws + ((static_cast<size_t>(seq) * a.heads + h) * a.segs + seg) * state_elems;   // used when segs > 1
  const float* from = kFull && a.segs > 1 ? mid : slot;
  const bool zero = !kFull || (a.segs == 1 && a.positions[r0] == 0);
  float s[MT][NS][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
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
  auto publish_state = [&]() {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int j = 0; j < NS; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          split2(s[mt][j][2 * r], s[mt][j][2 * r + 1], hi, lo);
          __nv_bfloat16* p = st_s + (d0 + mt * 16 + g + r * 8) * PV + s0 + j * 8 + q4 * 2;
          *reinterpret_cast<uint32_t*>(p) = hi;
          *reinterpret_cast<uint32_t*>(p + D * PV) = lo;
        }
  };
  if (kFull) publish_state();

  const int rw = warp & 3, o0 = (warp >> 2) * (VS / 2);   // output rows and columns of the warp
  const uint32_t a_off = ((rw * 16 + (lane & 15)) * PD + (lane >> 4) * 8) * 2;                          // Q rows of this warp
  const uint32_t b_off = (((lane & 7) + ((lane >> 4) << 3)) * PD + ((lane >> 3) & 1) * 8) * 2;          // K as [tokens][dims]
  const uint32_t t_off = (((lane & 7) + ((lane >> 3) & 1) * 8) * PV + (lane >> 4) * 8) * 2;             // [k][n] operands, transposed
  const uint32_t kt_off = (((lane & 7) + (lane >> 4) * 8) * PD + d0 + ((lane >> 3) & 1) * 8) * 2;       // K^T rows of this warp

  for (int c = 0; c < chunks; ++c) {
    const int b = c & 1, m = min(kChunk, n - c * kChunk);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                 // chunk c landed, state published, buffers of chunk c - 1 free
    issue(c + 1);
    const uint32_t kb = sm100::smem_u32(k_s + b * kChunk * PD);
    if constexpr (kFull) {
      const uint32_t qb = sm100::smem_u32(q_s + b * kChunk * PD) + a_off;
      const uint32_t vb = sm100::smem_u32(v_s + b * kChunk * PV) + t_off + o0 * 2;
      const uint32_t sb = sm100::smem_u32(st_s) + t_off + o0 * 2;
      float o[NO][4], p[8][4];
#pragma unroll
      for (int j = 0; j < NO; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) p[j][e] = 0.f;
      // S^T q, and the scores of this warp's rows against tokens up to its own
#pragma unroll 2
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t qa[4];
        ldsm4(qb + ks * 32, qa);
#pragma unroll
        for (int j = 0; j < 4; ++j) {                // 16 tokens each
          if (j <= rw) {
            uint32_t kf[4];
            ldsm4(kb + b_off + (j * 16 * PD + ks * 16) * 2, kf);
            mma(p[2 * j], qa, kf[0], kf[1]);
            mma(p[2 * j + 1], qa, kf[2], kf[3]);
          }
        }
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
      const float f0 = pw[i0 + 1], f1 = pw[i0 + 9];
#pragma unroll
      for (int j = 0; j < NO; ++j) o[j][0] *= f0, o[j][1] *= f0, o[j][2] *= f1, o[j][3] *= f1;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (j <= rw) {
          uint32_t ph[4], pl[4];
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int t = j * 16 + u * 8 + q4 * 2;
            auto w = [&](int i, int tok) { return tok <= i ? pw[i - tok] : 0.f; };
            split2(p[2 * j + u][0] * w(i0, t), p[2 * j + u][1] * w(i0, t + 1), ph[2 * u], pl[2 * u]);
            split2(p[2 * j + u][2] * w(i0 + 8, t), p[2 * j + u][3] * w(i0 + 8, t + 1), ph[2 * u + 1], pl[2 * u + 1]);
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
#pragma unroll
      for (int v = 0; v < NO; ++v) {
        const int col = c0 + o0 + v * 8 + q4 * 2;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int i = i0 + r * 8;
          if (i < m && col < a.vdim)                 // vdim is even
            *reinterpret_cast<float2*>(a.out + static_cast<size_t>(r0 + c * kChunk + i) * a.heads * a.vdim + h * a.vdim + col) =
                make_float2(o[v][2 * r], o[v][2 * r + 1]);
        }
      }
      if (c + 1 == chunks && !last) break;           // the next segment has its own start state
    }
    if (kFull) __syncthreads();                      // everyone is done with the published state
    const float pn = pw[m];
    const uint32_t vt = sm100::smem_u32(v_s + b * kChunk * PV) + t_off + s0 * 2;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int j = 0; j < NS; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[mt][j][e] *= pn;
#pragma unroll
    for (int kk = 0; kk < kChunk / 16; ++kk) {
      // keys of 16 tokens with their decay, as a bf16 pair
      const int t = kk * 16 + q4 * 2;
      auto w = [&](int tok) { return tok < m ? pw[m - 1 - tok] : 0.f; };
      const float w0 = w(t), w1 = w(t + 1), w8 = w(t + 8), w9 = w(t + 9);
      uint32_t hi[MT][4], lo[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        uint32_t ka[4];
        ldsm4t(kb + kt_off + (kk * 16 * PD + mt * 16) * 2, ka);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&ka[i]));
          split2(x.x * (i < 2 ? w0 : w8), x.y * (i < 2 ? w1 : w9), hi[mt][i], lo[mt][i]);
        }
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
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int d = d0 + mt * 16 + g + r * 8, c = c0 + s0 + j * 8 + q4 * 2;
        if (d < a.dim && c < a.vdim)
          *reinterpret_cast<float2*>(to + static_cast<size_t>(d) * a.vdim + c) = make_float2(s[mt][j][2 * r], s[mt][j][2 * r + 1]);
      }
}

// What each segment adds -> the state before each segment, in place.
__global__ void __launch_bounds__(256)
linear_scan_kernel(XpLinearAttnArgs a) {
  const int h = blockIdx.y, seq = blockIdx.z;
  const int total = a.q_lens[seq];
  if (total <= 0) return;
  const size_t state_elems = static_cast<size_t>(a.dim) * a.vdim;
  const size_t i = blockIdx.x * 256ull + threadIdx.x;
  if (i >= state_elems) return;
  float* mid = a.ws + (static_cast<size_t>(seq) * a.heads + h) * a.segs * state_elems + i;
  float x = a.positions[a.q_starts[seq]] == 0 ? 0.f : a.state[(static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * state_elems + i];
  const float p64 = a.decay_pow[h * (kChunk + 1) + kChunk];
  float f = 1.f;                                     // decay over one whole segment
  for (int c = 0; c < a.seg_tokens / kChunk; ++c) f *= p64;
  const int segs = (total + a.seg_tokens - 1) / a.seg_tokens;
  constexpr int kAhead = 8;                          // loads in flight before the first store
  for (int s0 = 0; s0 < segs; s0 += kAhead) {
    float add[kAhead];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) add[u] = s0 + u + 1 < segs ? mid[(s0 + u) * state_elems] : 0.f;   // the last segment adds to nobody
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      if (s0 + u >= segs) break;
      mid[(s0 + u) * state_elems] = x;
      x = fmaf(f, x, add[u]);
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

template <int D, int VS>
int launch_chunked(const XpLinearAttnArgs& a, cudaStream_t s) {
  constexpr int kSmem = chunk_smem_bytes<D, VS>();
  static_assert(kSmem <= 227 * 1024, "chunk buffers exceed the shared memory of an SM");
  int rc = big_smem(linear_chunked_kernel<D, VS, true>, kSmem);
  if (rc == 0) rc = big_smem(linear_chunked_kernel<D, VS, false>, kSmem);
  if (rc != 0) return rc;
  XpLinearAttnArgs b = a;
  if (b.segs <= 1) {
    b.segs = 1;
    b.seg_tokens = 0x40000000;
  } else if (b.ws == nullptr || b.seg_tokens <= 0 || b.seg_tokens % kChunk != 0) {
    return -13;
  }
  const dim3 grid((a.vdim + VS - 1) / VS * b.segs, a.heads, a.seqs);
  if (b.segs > 1) {
    linear_chunked_kernel<D, VS, false><<<grid, kChunkThreads, kSmem, s>>>(b);
    linear_scan_kernel<<<dim3((a.dim * a.vdim + 255) / 256, a.heads, a.seqs), 256, 0, s>>>(b);
  }
  linear_chunked_kernel<D, VS, true><<<grid, kChunkThreads, kSmem, s>>>(b);
  return done();
}

template <int D>
int launch_chunked_any(const XpLinearAttnArgs& a, cudaStream_t s) {
  if (a.vdim <= 32) return launch_chunked<D, 32>(a, s);
  if (a.vdim <= 64) return launch_chunked<D, 64>(a, s);
  return launch_chunked<D, 128>(a, s);
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

// Portion s: q_lens[s] rows from row q_starts[s]. segs > 1: every portion has at most segs * seg_tokens rows.
extern "C" int xp_linear_attn_prefill(const XpLinearAttnArgs* a, void* stream) {
  if (a->seqs <= 0) return 0;
  if (a->heads <= 0 || a->dim <= 0 || a->vdim <= 0) return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->f32) return launch_sequential_any<float>(*a, s);
  const bool chunked = !a->force_sequential && a->dim <= 256 && a->dim % 8 == 0 && a->vdim % 8 == 0 && a->ld_proj % 8 == 0 &&
                       a->q_off % 8 == 0 && a->k_off % 8 == 0 && a->v_off % 8 == 0 && reinterpret_cast<uintptr_t>(a->proj) % 16 == 0 &&
                       reinterpret_cast<uintptr_t>(a->out) % 8 == 0;
  if (!chunked) return launch_sequential_any<__nv_bfloat16>(*a, s);
  if (a->dim <= 64) return launch_chunked_any<64>(*a, s);
  if (a->dim <= 128) return launch_chunked_any<128>(*a, s);
  return launch_chunked<256, 32>(*a, s);
}
