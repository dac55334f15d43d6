// Gated delta rule over portions of prompts in chunks of 64 tokens on the tensor cores (bf16 rows, up to 128 key dimensions).
//
// With c_i the running sum of log g in a chunk, S the state before it, and the factors a_i (query), b_i (key) that make the
// rows unit vectors, all writes of a chunk solve one triangular system:
//   (1 + L) U = diag(beta) (V - R),   L_ij = beta_i b_i b_j e^(c_i - c_j) k_i . k_j  (j < i),   R_i = e^(c_i) b_i S^T k_i
//   o_i = e^(c_i) a_i S^T q_i + sum_{j <= i} M_ij u_j,   M_ij = a_i b_j e^(c_i - c_j) q_i . k_j
//   S  <- e^(c_n) S + sum_j k_j (b_j e^(c_n - c_j) u_j)^T
//   delta_chunk_kernel   per (chunk, head), all at once: T = (1 + L)^-1 diag(beta), M and the factors, to the workspace
//   delta_scan_kernel    per (16 or 32 value columns, head, sequence): walks the chunks with its part of the state in registers
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

// What the chunk kernel leaves for a (chunk, head).
struct __align__(16) Record {
  __nv_bfloat16 t[2][kChunk * kChunk];     // T: high parts, low parts
  __nv_bfloat16 m[2][kChunk * kChunk];
  float read_k[kChunk];                    // e^(c_i) b_i
  float read_q[kChunk];                    // e^(c_i) a_i
  float write[kChunk];                     // b_j e^(c_n - c_j)
  float decay[4];                          // e^(c_n), four times
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
    if (t < 4) rec->decay[t] = expf(cum[kChunk - 1]);
  }
  __syncthreads();
  // (1 + L)^-1 in halves of 32: the diagonal blocks by forward substitution (thread = column), T21 = -T22 (L21 T11) by all.
  constexpr int kHalf = 32, PT = kHalf + 1;
  float (*t_s)[kHalf][PT] = reinterpret_cast<float (*)[kHalf][PT]>(q_s);   // T11, T22, L21 T11, over the queries and keys
  if (warp < 2) {
    const float* base = l_s + warp * kHalf * PL + warp * kHalf;
    float x[kHalf];
#pragma unroll
    for (int i = 0; i < kHalf; ++i) {
      float s[4] = {i == lane ? 1.f : 0.f, 0.f, 0.f, 0.f};
      const float4* row = reinterpret_cast<const float4*>(base + i * PL);
#pragma unroll
      for (int m4 = 0; m4 < (i + 3) / 4; ++m4) {     // L is zero on and above the diagonal
        const float4 v = row[m4];
        s[0] = fmaf(-v.x, m4 * 4 < i ? x[m4 * 4] : 0.f, s[0]);
        s[1] = fmaf(-v.y, m4 * 4 + 1 < i ? x[m4 * 4 + 1] : 0.f, s[1]);
        s[2] = fmaf(-v.z, m4 * 4 + 2 < i ? x[m4 * 4 + 2] : 0.f, s[2]);
        s[3] = fmaf(-v.w, m4 * 4 + 3 < i ? x[m4 * 4 + 3] : 0.f, s[3]);
      }
      x[i] = (s[0] + s[1]) + (s[2] + s[3]);
      t_s[warp][i][lane] = x[i];
    }
  }
  __syncthreads();
  const int i1 = warp * 8;                           // eight rows of the lower left block, column = lane
  float x[8];
#pragma unroll
  for (int r = 0; r < 8; ++r) x[r] = 0.f;
#pragma unroll
  for (int m = 0; m < kHalf; m += 4) {
    const float y0 = t_s[0][m][lane], y1 = t_s[0][m + 1][lane], y2 = t_s[0][m + 2][lane], y3 = t_s[0][m + 3][lane];
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      const float4 v = *reinterpret_cast<const float4*>(l_s + (kHalf + i1 + r) * PL + m);
      x[r] = fmaf(v.x, y0, fmaf(v.y, y1, fmaf(v.z, y2, fmaf(v.w, y3, x[r]))));
    }
  }
#pragma unroll
  for (int r = 0; r < 8; ++r) t_s[2][i1 + r][lane] = x[r];
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 8; ++r) x[r] = 0.f;
#pragma unroll 8
  for (int m = 0; m < kHalf; ++m) {
    const float y = t_s[2][m][lane];
#pragma unroll
    for (int r = 0; r < 8; ++r) x[r] = fmaf(-t_s[1][i1 + r][m], y, x[r]);
  }
  auto store_t = [&](int i, int t, float v) {
    v *= beta[t];
    const __nv_bfloat16 hi = __float2bfloat16_rn(v);
    rec->t[0][i * kChunk + t] = hi;
    rec->t[1][i * kChunk + t] = __float2bfloat16_rn(v - __bfloat162float(hi));
  };
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    store_t(i1 + r, lane, t_s[0][i1 + r][lane]);
    store_t(kHalf + i1 + r, lane, x[r]);
    store_t(kHalf + i1 + r, kHalf + lane, t_s[1][i1 + r][lane]);
  }
}

template <int D, int VS>
struct ScanSmem {
  static constexpr int PD = D + 8, PV = VS + 8;
  __nv_bfloat16 q[2][kChunk * PD], k[2][kChunk * PD];
  __nv_bfloat16 t[2][2][kChunk * kPC], m[2][2][kChunk * kPC];
  __nv_bfloat16 s[2][2][D * PV];           // state before chunk c in buffer c & 1; high and low parts
  __nv_bfloat16 r[2][kChunk * PV];         // V - R
  __nv_bfloat16 w[2][kChunk * PV];         // writes, scaled for the state
  __nv_bfloat16 u[2][2][kChunk * PV];      // writes of chunk c in buffer c & 1
  float f[2][3][kChunk];
  float decay[2][4];
};

__device__ __forceinline__ void chain_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// B operands of one k-step (16 rows of a [k][n] tile of pitch PV) for a warp's NT column tiles. A single column tile takes two
// k-steps with one ldmatrix: every second call is free.
template <int NT, int PV>
struct BTile {
  uint32_t addr;
  uint32_t r[4];
  __device__ __forceinline__ BTile(const __nv_bfloat16* tile, int col, int lane) {
    addr = sm100::smem_u32(tile + col) + (NT == 2 ? bt_lane(lane, PV) : static_cast<uint32_t>(lane * PV * 2));
  }
  __device__ __forceinline__ void load(int ks) {
    if (NT == 2 || (ks & 1) == 0) ldsm4t(addr + ks * 16 * PV * 2, r);
  }
  __device__ __forceinline__ uint32_t b0(int j, int ks) const { return NT == 2 ? r[j * 2] : r[(ks & 1) * 2]; }
  __device__ __forceinline__ uint32_t b1(int j, int ks) const { return NT == 2 ? r[j * 2 + 1] : r[(ks & 1) * 2 + 1]; }
};

// Warps 0-7 carry the chain state -> V - R -> U -> state; warps 8-15 compute the outputs beside it: S^T q of the chunk at hand,
// and M U of the chunk before. In both groups a warp owns 16 tokens and half of the columns (the state: 16 of its rows).
template <int D, int VS>
__global__ void __launch_bounds__(512, 1)
delta_scan_kernel(XpDeltaArgs a) {
  using Smem = ScanSmem<D, VS>;
  constexpr int PD = Smem::PD, PV = Smem::PV;
  constexpr int NT = VS / 16;                        // column tiles of a warp
  constexpr int NS = D >= 128 ? VS / 8 : VS / 16;    // state column tiles of a warp; its 16 rows start at d0
  extern __shared__ __align__(16) uint8_t smem[];
  Smem& sm = *reinterpret_cast<Smem*>(smem);
  const int c0 = blockIdx.x * VS, h = blockIdx.y, seq = blockIdx.z;
  const int n = a.q_lens[seq];
  if (n <= 0) return;
  const int r0 = a.q_starts[seq], chunks = (n + kChunk - 1) / kChunk;
  const int hk = h / (a.heads / a.kv_heads), nq = a.kv_heads * a.dim, channels = 2 * nq + a.heads * a.vdim;
  const __nv_bfloat16* qkv = reinterpret_cast<const __nv_bfloat16*>(a.qkv) + static_cast<size_t>(r0) * channels;
  const Record* recs = reinterpret_cast<const Record*>(a.ws) + static_cast<size_t>(first_record(r0, seq)) * a.heads + h;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q4 = lane & 3;
  const bool chain = warp < 8;
  const int rw = warp & 3, col = ((warp >> 2) & 1) * (VS / 2);
  const int i0 = rw * 16 + g;                        // the lane's rows of a chunk: i0 and i0 + 8

  auto issue_matrix = [&](__nv_bfloat16 (&dst)[2][kChunk * kPC], const __nv_bfloat16 (&src)[2][kChunk * kChunk]) {
#pragma unroll
    for (int i = threadIdx.x - 256; i < 2 * kChunk * 8; i += 256) {
      const int p = i >> 9, t = (i >> 3) & 63, e = (i & 7) * 8;
      if (e / 16 <= t / 16) copy16(dst[p] + t * kPC + e, src[p] + t * kChunk + e, true);   // blocks above the diagonal are never read
    }
  };
  // rows, T and factors of chunk c, M of the chunk before; by the warps off the chain
  auto issue = [&](int c) {
    if (chain) return;
    if (c < chunks) {
      const int b = c & 1, m = min(kChunk, n - c * kChunk);
      const __nv_bfloat16* rows = qkv + static_cast<size_t>(c) * kChunk * channels + hk * a.dim;
      constexpr int kPieces = D / 8;
#pragma unroll
      for (int i = threadIdx.x - 256; i < kChunk * kPieces; i += 256) {
        const int t = i / kPieces, e = i % kPieces * 8;
        const bool ok = t < m && e < a.dim;
        const __nv_bfloat16* src = rows + static_cast<size_t>(ok ? t : 0) * channels + (ok ? e : 0);
        copy16(sm.q[b] + t * PD + e, src, ok);
        copy16(sm.k[b] + t * PD + e, src + nq, ok);
      }
      const Record* rec = recs + static_cast<size_t>(c) * a.heads;
      issue_matrix(sm.t[b], rec->t);
      const int i = threadIdx.x - 256;
      if (i < 48) copy16(&sm.f[b][0][0] + i * 4, rec->read_k + i * 4, true);     // three arrays in a row
      if (i == 64) copy16(sm.decay[b], rec->decay, true);
    }
    if (c > 0 && c <= chunks) issue_matrix(sm.m[(c - 1) & 1], recs[static_cast<size_t>(c - 1) * a.heads].m);
    copies_issued();
  };
  issue(0);

  // values of the lane's rows, one chunk ahead
  uint32_t v[NT][2];
  auto load_v = [&](int c) {
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = c * kChunk + i0 + r * 8, cc = c0 + col + j * 8 + q4 * 2;
        v[j][r] = t < n && cc < a.vdim ? *reinterpret_cast<const uint32_t*>(qkv + static_cast<size_t>(t) * channels + 2 * nq + h * a.vdim + cc) : 0u;
      }
  };
  const int d0 = D >= 128 ? (warp & 7) * 16 : rw * 16, s0 = D >= 128 ? 0 : col;
  float* slot = a.state + (static_cast<size_t>(a.state_slots[seq]) * a.heads + h) * a.dim * a.vdim;
  float s[NS][4];
  auto publish = [&](int b) {
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        uint32_t hi, lo;
        split2(s[j][2 * r], s[j][2 * r + 1], hi, lo);
        const int at = (d0 + g + r * 8) * PV + s0 + j * 8 + q4 * 2;
        *reinterpret_cast<uint32_t*>(sm.s[b][0] + at) = hi;
        *reinterpret_cast<uint32_t*>(sm.s[b][1] + at) = lo;
      }
  };
  if (chain) {
    load_v(0);
    const bool fresh = a.positions[r0] == 0;
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
    publish(0);
  }

  float o[NT][4];                                    // outputs of the chunk at hand until its M U joins them
  for (int c = 0; c <= chunks; ++c) {
    const int b = c & 1;
    copies_wait<0>();
    __syncthreads();                                 // chunk c landed, state published, writes of chunk c - 1 there
    issue(c + 1);
    if (!chain && c > 0) {
      // ---- o += M U, and out
      float x[2][NT][4];
#pragma unroll
      for (int p = 0; p < 2; ++p)
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) x[p][j][e] = p ? 0.f : o[j][e];
      const uint32_t m_hi = sm100::smem_u32(sm.m[b ^ 1][0] + rw * 16 * kPC) + a_lane(lane, kPC);
      const uint32_t m_lo = sm100::smem_u32(sm.m[b ^ 1][1] + rw * 16 * kPC) + a_lane(lane, kPC);
      BTile<NT, PV> uh(sm.u[b ^ 1][0], col, lane), ul(sm.u[b ^ 1][1], col, lane);
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks <= rw) {
          uint32_t mh[4], ml[4];
          ldsm4(m_hi + ks * 32, mh);
          ldsm4(m_lo + ks * 32, ml);
          uh.load(ks), ul.load(ks);
#pragma unroll
          for (int j = 0; j < NT; ++j) {
            mma(x[0][j], mh, uh.b0(j, ks), uh.b1(j, ks));
            mma(x[1][j], mh, ul.b0(j, ks), ul.b1(j, ks));
            mma(x[1][j], ml, uh.b0(j, ks), uh.b1(j, ks));
          }
        }
      }
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int cc = c0 + col + j * 8 + q4 * 2;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = (c - 1) * kChunk + i0 + r * 8;
          if (t < n && cc < a.vdim)
            *reinterpret_cast<float2*>(reinterpret_cast<float*>(a.out) + static_cast<size_t>(r0 + t) * a.ld_out + h * a.vdim + cc) =
                make_float2(x[0][j][2 * r] + x[1][j][2 * r], x[0][j][2 * r + 1] + x[1][j][2 * r + 1]);
        }
      }
    }
    if (c == chunks) break;
    // ---- S^T k (chain) and S^T q
    float y[2][NT][4];
#pragma unroll
    for (int p = 0; p < 2; ++p)
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[p][j][e] = 0.f;
    {
      const uint32_t rows_a = sm100::smem_u32((chain ? sm.k[b] : sm.q[b]) + rw * 16 * PD) + a_lane(lane, PD);
      BTile<NT, PV> sh(sm.s[b][0], col, lane), sl(sm.s[b][1], col, lane);
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t fa[4];
        ldsm4(rows_a + ks * 32, fa);
        sh.load(ks), sl.load(ks);
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          mma(y[0][j], fa, sh.b0(j, ks), sh.b1(j, ks));
          mma(y[1][j], fa, sl.b0(j, ks), sl.b1(j, ks));
        }
      }
    }
    const float f0 = sm.f[b][chain ? 0 : 1][i0], f1 = sm.f[b][chain ? 0 : 1][i0 + 8];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[j][e] = (y[0][j][e] + y[1][j][e]) * (e < 2 ? f0 : f1);
    if (!chain) continue;
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int at = (i0 + r * 8) * PV + col + j * 8 + q4 * 2;
        const float2 x = unpack2(v[j][r]);
        uint32_t hi, lo;
        split2(x.x - o[j][2 * r], x.y - o[j][2 * r + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(sm.r[0] + at) = hi;
        *reinterpret_cast<uint32_t*>(sm.r[1] + at) = lo;
      }
    load_v(c + 1);
    chain_sync();
    // ---- U = T (V - R)
#pragma unroll
    for (int p = 0; p < 2; ++p)
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[p][j][e] = 0.f;
    {
      const uint32_t t_hi = sm100::smem_u32(sm.t[b][0] + rw * 16 * kPC) + a_lane(lane, kPC);
      const uint32_t t_lo = sm100::smem_u32(sm.t[b][1] + rw * 16 * kPC) + a_lane(lane, kPC);
      BTile<NT, PV> rh(sm.r[0], col, lane), rl(sm.r[1], col, lane);
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks <= rw) {
          uint32_t th[4], tl[4];
          ldsm4(t_hi + ks * 32, th);
          ldsm4(t_lo + ks * 32, tl);
          rh.load(ks), rl.load(ks);
#pragma unroll
          for (int j = 0; j < NT; ++j) {
            mma(y[0][j], th, rh.b0(j, ks), rh.b1(j, ks));
            mma(y[1][j], th, rl.b0(j, ks), rl.b1(j, ks));
            mma(y[1][j], tl, rh.b0(j, ks), rh.b1(j, ks));
          }
        }
      }
    }
    const float w0 = sm.f[b][2][i0], w1 = sm.f[b][2][i0 + 8];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int at = (i0 + r * 8) * PV + col + j * 8 + q4 * 2;
        const float x0 = y[0][j][2 * r] + y[1][j][2 * r], x1 = y[0][j][2 * r + 1] + y[1][j][2 * r + 1], w = r ? w1 : w0;
        uint32_t hi, lo;
        split2(x0 * w, x1 * w, hi, lo);
        *reinterpret_cast<uint32_t*>(sm.w[0] + at) = hi;
        *reinterpret_cast<uint32_t*>(sm.w[1] + at) = lo;
        split2(x0, x1, hi, lo);
        *reinterpret_cast<uint32_t*>(sm.u[b][0] + at) = hi;
        *reinterpret_cast<uint32_t*>(sm.u[b][1] + at) = lo;
      }
    chain_sync();
    // ---- state
    const float dec = sm.decay[b][0];
    const uint32_t kt = sm100::smem_u32(sm.k[b] + d0) + at_lane(lane, PD);
    const uint32_t w_hi = sm100::smem_u32(sm.w[0] + s0) + bt_lane(lane, PV), w_lo = sm100::smem_u32(sm.w[1] + s0) + bt_lane(lane, PV);
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[j][e] *= dec;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t ka[4];
      ldsm4t(kt + ks * 16 * PD * 2, ka);
      if constexpr (NS == 1) {
        uint32_t bh[4], bl[4];             // (the second tile belongs to the other half's warp)
        ldsm4t(w_hi + ks * 16 * PV * 2 - (s0 ? 16 : 0), bh);
        ldsm4t(w_lo + ks * 16 * PV * 2 - (s0 ? 16 : 0), bl);
        mma(s[0], ka, s0 ? bh[2] : bh[0], s0 ? bh[3] : bh[1]);
        mma(s[0], ka, s0 ? bl[2] : bl[0], s0 ? bl[3] : bl[1]);
      } else {
#pragma unroll
        for (int j = 0; j < NS; j += 2) {
          uint32_t bh[4], bl[4];
          ldsm4t(w_hi + (ks * 16 * PV + j * 8) * 2, bh);
          ldsm4t(w_lo + (ks * 16 * PV + j * 8) * 2, bl);
          mma(s[j], ka, bh[0], bh[1]);
          mma(s[j + 1], ka, bh[2], bh[3]);
          mma(s[j], ka, bl[0], bl[1]);
          mma(s[j + 1], ka, bl[2], bl[3]);
        }
      }
    }
    if (c + 1 < chunks) publish(b ^ 1);
  }
  copies_wait<0>();
  if (!chain) return;
#pragma unroll
  for (int j = 0; j < NS; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + g + r * 8, c = c0 + s0 + j * 8 + q4 * 2;
      if (d < a.dim && c < a.vdim)
        *reinterpret_cast<float2*>(slot + static_cast<size_t>(d) * a.vdim + c) = make_float2(s[j][2 * r], s[j][2 * r + 1]);
    }
}

template <int D, int VS>
int launch_scan(const XpDeltaArgs& a, cudaStream_t s) {
  constexpr int kBytes = sizeof(ScanSmem<D, VS>);
  static_assert(kBytes <= 227 * 1024, "tiles exceed the shared memory of an SM");
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(delta_scan_kernel<D, VS>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes) != cudaSuccess) return -21;
    attr_set = true;
  }
  delta_scan_kernel<D, VS><<<dim3((a.vdim + VS - 1) / VS, a.heads, a.seqs), 512, kBytes, s>>>(a);
  return 0;
}

template <int D>
int launch(const XpDeltaArgs& a, cudaStream_t s) {
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(delta_chunk_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, chunk_smem<D>()) != cudaSuccess) return -21;
    attr_set = true;
  }
  delta_chunk_kernel<D><<<dim3((a.max_q + kChunk - 1) / kChunk, a.heads, a.seqs), 128, chunk_smem<D>(), s>>>(a);
  // narrow columns while they still fit on the SMs at the same time
  const bool narrow = static_cast<int64_t>((a.vdim + 15) / 16) * a.heads * a.seqs <= 148;
  const int rc = narrow ? launch_scan<D, 16>(a, s) : launch_scan<D, 32>(a, s);
  if (rc != 0) return rc;
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
