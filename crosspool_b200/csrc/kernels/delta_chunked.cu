// Gated delta rule over portions of prompts in chunks of 64 tokens on the tensor cores (bf16 rows, up to 128 key dimensions).
//
// With c_i the running sum of log g in a chunk, S the state before it, and the factors a_i (query), b_i (key) that make the
// rows unit vectors, all writes of a chunk solve one triangular system:
//   (1 + L) U = diag(beta) (V - R),   L_ij = beta_i b_i b_j e^(c_i - c_j) k_i . k_j  (j < i),   R_i = e^(c_i) b_i S^T k_i
//   o_i = e^(c_i) a_i S^T q_i + sum_{j <= i} M_ij u_j,   M_ij = a_i b_j e^(c_i - c_j) q_i . k_j
//   S  <- e^(c_n) S + sum_j k_j (b_j e^(c_n - c_j) u_j)^T
//   delta_chunk_kernel   per (chunk, head), all at once: T = (1 + L)^-1 diag(beta), M and the factors, to the workspace
//   delta_scan_kernel    per (32 value columns, head, sequence): walks the chunks with its part of the state in registers
// Queries and keys enter their products as the bf16 rows they are, their factors in fp32 afterwards; T, M, U and the state
// enter as bf16 pairs (high and low part), so that everything of the recurrence keeps at least 16 mantissa bits.
//
// mma.sync rather than tcgen05: the state and U have to be scaled and split again several times per chunk, which from tensor
// memory costs a round trip each.
#include "xpool/mixer_api.h"
#include "xpool/mma_sync.cuh"

namespace xpool {
namespace delta {

using namespace xpool::frag;

constexpr int kChunk = 64;
constexpr int kPC = kChunk + 8;            // pitch of chunk x chunk tiles
constexpr int kVS = 32;                    // value columns of a scanning CTA
constexpr int kPV = kVS + 8;

// What the chunk kernel leaves for a (chunk, head).
struct __align__(16) Record {
  __nv_bfloat16 t[2][kChunk * kChunk];     // T: high parts, low parts
  __nv_bfloat16 m[2][kChunk * kChunk];
  float read_k[kChunk];                    // e^(c_i) b_i
  float read_q[kChunk];                    // e^(c_i) a_i
  float write[kChunk];                     // b_j e^(c_n - c_j)
  float decay[4];                          // e^(c_n)
};

// Records of a sequence start here: distinct for all chunks of a batch of packed portions.
__device__ __forceinline__ int first_record(int start, int seq) { return start / kChunk + seq; }

template <int D>
constexpr int chunk_smem() { return 2 * kChunk * (D + 8) * 2 + kChunk * (kChunk + 4) * 4; }

template <int D>
__global__ void __launch_bounds__(128)
delta_chunk_kernel(XpDeltaArgs a) {
  constexpr int PD = D + 8, PL = kChunk + 4;
  extern __shared__ __align__(16) uint8_t smem[];
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* k_s = q_s + kChunk * PD;
  float* l_s = reinterpret_cast<float*>(k_s + kChunk * PD);          // L, row-major
  __shared__ float cum[kChunk], fa[kChunk], fb[kChunk], beta[kChunk];
  const int h = blockIdx.y, seq = blockIdx.z, total = a.q_lens[seq];
  const int t0 = blockIdx.x * kChunk;
  if (t0 >= total) return;
  const int n = min(kChunk, total - t0), r0 = a.q_starts[seq] + t0;
  const int hk = h / (a.heads / a.kv_heads), nq = a.kv_heads * a.dim, channels = 2 * nq + a.heads * a.vdim;
  const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(a.qkv) + static_cast<size_t>(r0) * channels + hk * a.dim;
  constexpr int kPieces = D / 8;
  for (int i = threadIdx.x; i < kChunk * kPieces; i += 128) {
    const int t = i / kPieces, e = i % kPieces * 8;
    const bool ok = t < n && e < a.dim;
    const __nv_bfloat16* src = rows + static_cast<size_t>(ok ? t : 0) * channels + (ok ? e : 0);
    copy16(q_s + t * PD + e, src, ok);
    copy16(k_s + t * PD + e, src + nq, ok);
  }
  copies_issued();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q4 = lane & 3;
  if (threadIdx.x < kChunk) {
    const int t = threadIdx.x;
    const bool ok = t < n;                 // rows behind the portion: no decay, nothing written
    const size_t row = r0 + (ok ? t : 0);
    beta[t] = ok ? a.beta_g[row * 2 * a.heads + h] : 0.f;
    cum[t] = ok ? a.beta_g[row * 2 * a.heads + a.heads + h] : 0.f;
    fa[t] = ok ? a.qk_scale[row * 2 * a.kv_heads + hk] : 0.f;
    fb[t] = ok ? a.qk_scale[row * 2 * a.kv_heads + a.kv_heads + hk] : 0.f;
  }
  __syncthreads();
  if (warp == 0) {                         // running sums of log g: two per lane
    float x = cum[2 * lane], y = x + cum[2 * lane + 1], s = y;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float u = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += u;
    }
    cum[2 * lane] = s - y + x;
    cum[2 * lane + 1] = s;
  }
  copies_wait<0>();
  __syncthreads();

  Record* rec = reinterpret_cast<Record*>(a.ws) + static_cast<size_t>(first_record(a.q_starts[seq], seq) + blockIdx.x) * a.heads + h;
  // warp: 16 rows; products with the tokens of its own and earlier 16-token blocks
  float kk[8][4], qk[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) kk[j][e] = qk[j][e] = 0.f;
  const uint32_t ka = sm100::smem_u32(k_s + warp * 16 * PD) + a_lane(lane, PD), qa = sm100::smem_u32(q_s + warp * 16 * PD) + a_lane(lane, PD);
  const uint32_t kb = sm100::smem_u32(k_s) + b_lane(lane, PD);
#pragma unroll 2
  for (int ks = 0; ks < D / 16; ++ks) {
    uint32_t fk[4], fq[4];
    ldsm4(ka + ks * 32, fk);
    ldsm4(qa + ks * 32, fq);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (j <= warp) {
        uint32_t b[4];
        ldsm4(kb + (j * 16 * PD + ks * 16) * 2, b);
        mma(kk[2 * j], fk, b[0], b[1]);
        mma(kk[2 * j + 1], fk, b[2], b[3]);
        mma(qk[2 * j], fq, b[0], b[1]);
        mma(qk[2 * j + 1], fq, b[2], b[3]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = warp * 16 + g + r * 8;
    const float ci = cum[i], ai = fa[i], bi = fb[i] * beta[i];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      float l[2], m[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = j * 8 + q4 * 2 + e;
        const float f = t <= i ? expf(ci - cum[t]) * fb[t] : 0.f;
        l[e] = t < i ? f * bi * kk[j][2 * r + e] : 0.f;
        m[e] = f * ai * qk[j][2 * r + e];
      }
      const int at = j * 8 + q4 * 2;
      *reinterpret_cast<float2*>(l_s + i * PL + at) = make_float2(l[0], l[1]);
      uint32_t hi, lo;
      split2(m[0], m[1], hi, lo);
      *reinterpret_cast<uint32_t*>(rec->m[0] + i * kChunk + at) = hi;
      *reinterpret_cast<uint32_t*>(rec->m[1] + i * kChunk + at) = lo;
    }
  }
  if (threadIdx.x < kChunk) {
    const int t = threadIdx.x;
    const float e = expf(cum[t]);
    rec->read_k[t] = e * fb[t];
    rec->read_q[t] = e * fa[t];
    rec->write[t] = fb[t] * expf(cum[kChunk - 1] - cum[t]);
    if (t == 0) rec->decay[0] = expf(cum[kChunk - 1]);
  }
  __syncthreads();
  // Column t of (1 + L)^-1 by forward substitution, thread = column.
  if (threadIdx.x < kChunk) {
    const int t = threadIdx.x;
    float x[kChunk];
#pragma unroll
    for (int i = 0; i < kChunk; ++i) {
      float s[4] = {i == t ? 1.f : 0.f, 0.f, 0.f, 0.f};
      const float4* row = reinterpret_cast<const float4*>(l_s + i * PL);
#pragma unroll
      for (int m4 = 0; m4 < (i + 3) / 4; ++m4) {     // L is zero on and above the diagonal
        const float4 v = row[m4];
        s[0] = fmaf(-v.x, m4 * 4 < i ? x[m4 * 4] : 0.f, s[0]);
        s[1] = fmaf(-v.y, m4 * 4 + 1 < i ? x[m4 * 4 + 1] : 0.f, s[1]);
        s[2] = fmaf(-v.z, m4 * 4 + 2 < i ? x[m4 * 4 + 2] : 0.f, s[2]);
        s[3] = fmaf(-v.w, m4 * 4 + 3 < i ? x[m4 * 4 + 3] : 0.f, s[3]);
      }
      x[i] = (s[0] + s[1]) + (s[2] + s[3]);
    }
    const float b = beta[t];
#pragma unroll
    for (int i = 0; i < kChunk; ++i) {
      const float v = x[i] * b;
      const __nv_bfloat16 hi = __float2bfloat16_rn(v);
      rec->t[0][i * kChunk + t] = hi;
      rec->t[1][i * kChunk + t] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
  }
}

template <int D>
struct ScanSmem {
  static constexpr int PD = D + 8;
  __nv_bfloat16 q[2][kChunk * PD], k[2][kChunk * PD], v[2][kChunk * kPV];
  __nv_bfloat16 t[2][2][kChunk * kPC], m[2][2][kChunk * kPC];
  __nv_bfloat16 s[2][D * kPV];             // state, high and low parts
  __nv_bfloat16 r[2][kChunk * kPV];        // V - R, then the writes scaled for the state
  __nv_bfloat16 u[2][kChunk * kPV];
  float f[2][3][kChunk];
  float decay[2];
};

// Warps 0-3 work on keys (16 rows each), warps 4-7 on queries where the two differ.
template <int D>
__global__ void __launch_bounds__(256, 1)
delta_scan_kernel(XpDeltaArgs a) {
  constexpr int PD = D + 8;
  constexpr int NS = D >= 128 ? kVS / 8 : kVS / 16;  // state column tiles of a warp; its 16 rows start at d0
  extern __shared__ __align__(16) uint8_t smem[];
  ScanSmem<D>& sm = *reinterpret_cast<ScanSmem<D>*>(smem);
  const int c0 = blockIdx.x * kVS, h = blockIdx.y, seq = blockIdx.z;
  const int n = a.q_lens[seq];
  if (n <= 0) return;
  const int r0 = a.q_starts[seq], chunks = (n + kChunk - 1) / kChunk;
  const int hk = h / (a.heads / a.kv_heads), nq = a.kv_heads * a.dim, channels = 2 * nq + a.heads * a.vdim;
  const __nv_bfloat16* qkv = reinterpret_cast<const __nv_bfloat16*>(a.qkv) + static_cast<size_t>(r0) * channels;
  const Record* recs = reinterpret_cast<const Record*>(a.ws) + static_cast<size_t>(first_record(r0, seq)) * a.heads + h;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q4 = lane & 3;

  auto issue = [&](int c) {
    if (c < chunks) {
      const int b = c & 1, m = min(kChunk, n - c * kChunk);
      const __nv_bfloat16* rows = qkv + static_cast<size_t>(c) * kChunk * channels;
      constexpr int kPieces = D / 8;
#pragma unroll
      for (int i = threadIdx.x; i < kChunk * kPieces; i += 256) {
        const int t = i / kPieces, e = i % kPieces * 8;
        const bool ok = t < m && e < a.dim;
        const __nv_bfloat16* src = rows + static_cast<size_t>(ok ? t : 0) * channels + hk * a.dim + (ok ? e : 0);
        copy16(sm.q[b] + t * PD + e, src, ok);
        copy16(sm.k[b] + t * PD + e, src + nq, ok);
      }
      {
        const int t = threadIdx.x >> 2, e = (threadIdx.x & 3) * 8;
        const bool ok = t < m && c0 + e < a.vdim;
        copy16(sm.v[b] + t * kPV + e, rows + static_cast<size_t>(ok ? t : 0) * channels + 2 * nq + h * a.vdim + (ok ? c0 + e : 0), ok);
      }
      const Record* rec = recs + static_cast<size_t>(c) * a.heads;
#pragma unroll
      for (int p = 0; p < 2; ++p)
#pragma unroll
        for (int i = threadIdx.x; i < kChunk * 8; i += 256) {
          const int t = i >> 3, e = (i & 7) * 8;
          const bool ok = e / 16 <= t / 16;                  // blocks above the diagonal are never read
          if (ok) {
            copy16(sm.t[b][p] + t * kPC + e, rec->t[p] + t * kChunk + e, true);
            copy16(sm.m[b][p] + t * kPC + e, rec->m[p] + t * kChunk + e, true);
          }
        }
      if (threadIdx.x < 48) copy16(&sm.f[b][0][0] + threadIdx.x * 4, rec->read_k + threadIdx.x * 4, true);   // three arrays in a row
      if (threadIdx.x == 64) sm.decay[b] = rec->decay[0];
    }
    copies_issued();
  };
  issue(0);

  const int d0 = D >= 128 ? warp * 16 : (warp & 3) * 16, s0 = D >= 128 ? 0 : (warp >> 2) * (kVS / 2);
  float* slot = a.state + (static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * a.dim * a.vdim;
  const bool fresh = a.positions[r0] == 0;
  float s[NS][4];
#pragma unroll
  for (int j = 0; j < NS; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + g + r * 8, c = c0 + s0 + j * 8 + q4 * 2;
      float2 x = make_float2(0.f, 0.f);
      if (!fresh && d < a.dim && c < a.vdim) x = *reinterpret_cast<const float2*>(slot + static_cast<size_t>(d) * a.vdim + c);
      s[j][2 * r] = x.x;
      s[j][2 * r + 1] = x.y;
    }
  auto publish = [&](__nv_bfloat16 (&dst)[2][D * kPV]) {
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        uint32_t hi, lo;
        split2(s[j][2 * r], s[j][2 * r + 1], hi, lo);
        const int at = (d0 + g + r * 8) * kPV + s0 + j * 8 + q4 * 2;
        *reinterpret_cast<uint32_t*>(dst[0] + at) = hi;
        *reinterpret_cast<uint32_t*>(dst[1] + at) = lo;
      }
  };
  publish(sm.s);

  const int rw = warp & 3;
  const bool on_q = warp >= 4;
  const uint32_t bt_v = bt_lane(lane, kPV);
  const uint32_t s_hi = sm100::smem_u32(sm.s[0]) + bt_v, s_lo = sm100::smem_u32(sm.s[1]) + bt_v;
  const uint32_t r_hi = sm100::smem_u32(sm.r[0]) + bt_v, r_lo = sm100::smem_u32(sm.r[1]) + bt_v;
  const uint32_t u_hi = sm100::smem_u32(sm.u[0]) + bt_v, u_lo = sm100::smem_u32(sm.u[1]) + bt_v;
  for (int c = 0; c < chunks; ++c) {
    const int b = c & 1, m = min(kChunk, n - c * kChunk);
    copies_wait<0>();
    __syncthreads();                       // chunk c landed, state published, buffers of chunk c - 1 free
    issue(c + 1);
    // ---- S^T k and S^T q: warp = 16 rows, all columns
    float o[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
    const uint32_t rows_a = sm100::smem_u32((on_q ? sm.q[b] : sm.k[b]) + rw * 16 * PD) + a_lane(lane, PD);
#pragma unroll 4
    for (int ks = 0; ks < D / 16; ++ks) {
      uint32_t fa[4], h0[4], h1[4], l0[4], l1[4];
      ldsm4(rows_a + ks * 32, fa);
      ldsm4t(s_hi + ks * 16 * kPV * 2, h0);
      ldsm4t(s_hi + (ks * 16 * kPV + 16) * 2, h1);
      ldsm4t(s_lo + ks * 16 * kPV * 2, l0);
      ldsm4t(s_lo + (ks * 16 * kPV + 16) * 2, l1);
      mma(o[0], fa, h0[0], h0[1]);
      mma(o[1], fa, h0[2], h0[3]);
      mma(o[2], fa, h1[0], h1[1]);
      mma(o[3], fa, h1[2], h1[3]);
      mma(o[0], fa, l0[0], l0[1]);
      mma(o[1], fa, l0[2], l0[3]);
      mma(o[2], fa, l1[0], l1[1]);
      mma(o[3], fa, l1[2], l1[3]);
    }
    const int i0 = rw * 16 + g;            // rows i0 and i0 + 8 of the chunk
    {
      const float* f = sm.f[b][on_q ? 1 : 0];
      const float f0 = f[i0], f1 = f[i0 + 8];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        o[j][0] *= f0, o[j][1] *= f0, o[j][2] *= f1, o[j][3] *= f1;
        if (!on_q) {
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int at = (i0 + r * 8) * kPV + j * 8 + q4 * 2;
            const float2 v = unpack2(*reinterpret_cast<const uint32_t*>(sm.v[b] + at));
            uint32_t hi, lo;
            split2(v.x - o[j][2 * r], v.y - o[j][2 * r + 1], hi, lo);
            *reinterpret_cast<uint32_t*>(sm.r[0] + at) = hi;
            *reinterpret_cast<uint32_t*>(sm.r[1] + at) = lo;
          }
        }
      }
    }
    __syncthreads();
    // ---- U = T (V - R): warp = 16 rows, half of the columns
    float u[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) u[j][e] = 0.f;
    const int uc = (warp >> 2) * 16;
    const uint32_t ta_hi = sm100::smem_u32(sm.t[b][0] + rw * 16 * kPC) + a_lane(lane, kPC);
    const uint32_t ta_lo = sm100::smem_u32(sm.t[b][1] + rw * 16 * kPC) + a_lane(lane, kPC);
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      if (ks <= rw) {
        uint32_t th[4], tl[4], bh[4], bl[4];
        ldsm4(ta_hi + ks * 32, th);
        ldsm4(ta_lo + ks * 32, tl);
        ldsm4t(r_hi + (ks * 16 * kPV + uc) * 2, bh);
        ldsm4t(r_lo + (ks * 16 * kPV + uc) * 2, bl);
        mma(u[0], th, bh[0], bh[1]);
        mma(u[1], th, bh[2], bh[3]);
        mma(u[0], th, bl[0], bl[1]);
        mma(u[1], th, bl[2], bl[3]);
        mma(u[0], tl, bh[0], bh[1]);
        mma(u[1], tl, bh[2], bh[3]);
      }
    }
    __syncthreads();                       // everyone has read V - R
    {
      const float w0 = sm.f[b][2][i0], w1 = sm.f[b][2][i0 + 8];
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int at = (i0 + r * 8) * kPV + uc + j * 8 + q4 * 2;
          const float x = u[j][2 * r], y = u[j][2 * r + 1], w = r ? w1 : w0;
          uint32_t hi, lo;
          split2(x, y, hi, lo);
          *reinterpret_cast<uint32_t*>(sm.u[0] + at) = hi;
          *reinterpret_cast<uint32_t*>(sm.u[1] + at) = lo;
          split2(x * w, y * w, hi, lo);
          *reinterpret_cast<uint32_t*>(sm.r[0] + at) = hi;
          *reinterpret_cast<uint32_t*>(sm.r[1] + at) = lo;
        }
    }
    __syncthreads();
    // ---- outputs (warps of the queries)
    if (on_q) {
      const uint32_t ma_hi = sm100::smem_u32(sm.m[b][0] + rw * 16 * kPC) + a_lane(lane, kPC);
      const uint32_t ma_lo = sm100::smem_u32(sm.m[b][1] + rw * 16 * kPC) + a_lane(lane, kPC);
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks <= rw) {
          uint32_t mh[4], ml[4];
          ldsm4(ma_hi + ks * 32, mh);
          ldsm4(ma_lo + ks * 32, ml);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            uint32_t bh[4], bl[4];
            ldsm4t(u_hi + (ks * 16 * kPV + j * 16) * 2, bh);
            ldsm4t(u_lo + (ks * 16 * kPV + j * 16) * 2, bl);
            mma(o[2 * j], mh, bh[0], bh[1]);
            mma(o[2 * j + 1], mh, bh[2], bh[3]);
            mma(o[2 * j], mh, bl[0], bl[1]);
            mma(o[2 * j + 1], mh, bl[2], bl[3]);
            mma(o[2 * j], ml, bh[0], bh[1]);
            mma(o[2 * j + 1], ml, bh[2], bh[3]);
          }
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int col = c0 + j * 8 + q4 * 2;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int i = i0 + r * 8;
          if (i < m && col < a.vdim)
            *reinterpret_cast<float2*>(reinterpret_cast<float*>(a.out) + static_cast<size_t>(r0 + c * kChunk + i) * a.ld_out + h * a.vdim + col) =
                make_float2(o[j][2 * r], o[j][2 * r + 1]);
        }
      }
    }
    // ---- state: warp = 16 rows of it
    const float dec = sm.decay[b];
    const uint32_t kt = sm100::smem_u32(sm.k[b] + d0) + at_lane(lane, PD);
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[j][e] *= dec;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t ka[4];
      ldsm4t(kt + ks * 16 * PD * 2, ka);
#pragma unroll
      for (int j = 0; j < NS; j += 2) {
        uint32_t bh[4], bl[4];
        ldsm4t(r_hi + (ks * 16 * kPV + s0 + j * 8) * 2, bh);
        ldsm4t(r_lo + (ks * 16 * kPV + s0 + j * 8) * 2, bl);
        mma(s[j], ka, bh[0], bh[1]);
        mma(s[j + 1], ka, bh[2], bh[3]);
        mma(s[j], ka, bl[0], bl[1]);
        mma(s[j + 1], ka, bl[2], bl[3]);
      }
    }
    if (c + 1 < chunks) publish(sm.s);     // the reads of the old state lie two barriers back
  }
#pragma unroll
  for (int j = 0; j < NS; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + g + r * 8, c = c0 + s0 + j * 8 + q4 * 2;
      if (d < a.dim && c < a.vdim)
        *reinterpret_cast<float2*>(slot + static_cast<size_t>(d) * a.vdim + c) = make_float2(s[j][2 * r], s[j][2 * r + 1]);
    }
}

template <int D>
int launch(const XpDeltaArgs& a, cudaStream_t s) {
  static_assert(sizeof(ScanSmem<D>) <= 227 * 1024, "tiles exceed the shared memory of an SM");
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(delta_chunk_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, chunk_smem<D>()) != cudaSuccess ||
        cudaFuncSetAttribute(delta_scan_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, sizeof(ScanSmem<D>)) != cudaSuccess)
      return -21;
    attr_set = true;
  }
  delta_chunk_kernel<D><<<dim3((a.max_q + kChunk - 1) / kChunk, a.heads, a.seqs), 128, chunk_smem<D>(), s>>>(a);
  delta_scan_kernel<D><<<dim3((a.vdim + kVS - 1) / kVS, a.heads, a.seqs), 256, sizeof(ScanSmem<D>), s>>>(a);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -100 - static_cast<int>(e);
}

}  // namespace delta
}  // namespace xpool

// Bytes of workspace for batches of at most `rows` rows in `seqs` portions.
extern "C" size_t xp_delta_ws_bytes(int rows, int seqs, int heads) {
  return (static_cast<size_t>(rows) / xpool::delta::kChunk + seqs + 1) * heads * sizeof(xpool::delta::Record);
}

// Returns 1 when the sizes are outside what the chunked kernels cover, 0 when they were launched.
extern "C" int xp_delta_chunked(const XpDeltaArgs* a, void* stream) {
  const bool ok = !a->f32 && a->ws != nullptr && a->dim <= 128 && a->dim % 8 == 0 && a->vdim % 8 == 0 && a->ld_out % 2 == 0 &&
                  reinterpret_cast<uintptr_t>(a->qkv) % 16 == 0 && reinterpret_cast<uintptr_t>(a->ws) % 16 == 0 &&
                  reinterpret_cast<uintptr_t>(a->out) % 8 == 0 && reinterpret_cast<uintptr_t>(a->state) % 8 == 0;
  if (!ok) return 1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->dim <= 64 ? xpool::delta::launch<64>(*a, s) : xpool::delta::launch<128>(*a, s);
}
