// Plain fp32 matrix product y = x w^T (+ bias) for models served in 32-bit: FFMA only, no reduced-precision tensor mode.
// One CTA computes a 64 x 64 tile from 16-deep slices staged in shared memory; a thread owns 4 x 4 outputs.
#include <cuda_runtime.h>
#include <stdint.h>

#include "xpool/mixer_api.h"

namespace {

constexpr int kBM = 64, kBN = 64, kBK = 16;

// Rows r0 .. and features n0 .. of one product; rows and n bound both.
__device__ __forceinline__ void tile_f32(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ bias,
                                         float* __restrict__ out, int r0, int n0, int rows, int n, int k, int ldx, int ldw, int ldo, float scale,
                                         int silu_cols) {
  __shared__ float xs[kBK][kBM + 4];
  __shared__ float ws[kBK][kBN + 4];
  const int tr = threadIdx.x >> 4, tc = threadIdx.x & 15;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < k; k0 += kBK) {
    for (int i = threadIdx.x; i < kBM * kBK; i += 256) {
      const int kk = i & (kBK - 1), m = i / kBK;
      const bool kin = k0 + kk < k;
      xs[kk][m] = kin && r0 + m < rows ? x[static_cast<int64_t>(r0 + m) * ldx + k0 + kk] : 0.f;
      ws[kk][m] = kin && n0 + m < n ? w[static_cast<int64_t>(n0 + m) * ldw + k0 + kk] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kBK; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) a[j] = xs[kk][tr * 4 + j], b[j] = ws[kk][tc * 4 + j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = r0 + tr * 4 + i;
    if (r >= rows) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + tc * 4 + j;
      if (c >= n) continue;
      float v = fmaf(acc[i][j], scale, bias != nullptr ? bias[c] : 0.f);
      if (c < silu_cols) v = v / (1.f + expf(-v));
      out[static_cast<int64_t>(r) * ldo + c] = v;
    }
  }
}

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ bias, float* __restrict__ out,
                int rows, int n, int k, int ldx, int ldw, int ldo, int64_t sx, int64_t sw, int64_t so, float scale, int silu_cols) {
  tile_f32(x + blockIdx.z * sx, w + blockIdx.z * sw, bias, out + blockIdx.z * so, blockIdx.y * kBM, blockIdx.x * kBN, rows, n, k, ldx, ldw, ldo,
           scale, silu_cols);
}

// Grouped form: tiles {group, first feature of 128, first row, row end} of at most kBM rows from a device table; a CTA takes
// one half of a tile's features.
__global__ void __launch_bounds__(256)
gemm_f32_grouped_kernel(const float* __restrict__ x, const float* __restrict__ w, float* __restrict__ out, const int4* __restrict__ tiles,
                        const int* __restrict__ n_tiles, int n, int k, int ldx, int ldw, int ldo, int w_rows_per_group) {
  if (static_cast<int>(blockIdx.x) >= *n_tiles) return;
  const int4 t = tiles[blockIdx.x];
  const int n0 = t.y + blockIdx.y * kBN;
  if (n0 >= n) return;
  tile_f32(x, w + static_cast<int64_t>(t.x) * w_rows_per_group * ldw, nullptr, out, t.z, n0, min(t.w, t.z + kBM), n, k, ldx, ldw, ldo, 1.f, 0);
}

}  // namespace

extern "C" int xp_gemm_f32_grouped(const float* x, const float* w, float* out, const void* tiles, const int* n_tiles, int max_tiles, int n, int k,
                                   int ldx, int ldw, int ldo, int w_rows_per_group, void* stream) {
  if (max_tiles <= 0 || n <= 0) return 0;
  if (k <= 0) return -10;
  gemm_f32_grouped_kernel<<<dim3(max_tiles, 128 / kBN), 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(
      x, w, out, static_cast<const int4*>(tiles), n_tiles, n, k, ldx, ldw, ldo, w_rows_per_group);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -100 - static_cast<int>(e);
}

extern "C" int xp_gemm_f32(const float* x, const float* w, const float* bias, float* out, int rows, int n, int k, int ldx, int ldw,
                           int ldo, int batch, int64_t sx, int64_t sw, int64_t so, float out_scale, int silu_cols, void* stream) {
  if (rows <= 0 || n <= 0 || batch <= 0) return 0;
  if (k <= 0) return -10;
  dim3 grid((n + kBN - 1) / kBN, (rows + kBM - 1) / kBM, batch);
  gemm_f32_kernel<<<grid, 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(x, w, bias, out, rows, n, k, ldx, ldw, ldo, sx, sw, so,
                                                                           out_scale == 0.f ? 1.f : out_scale, silu_cols);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -100 - static_cast<int>(e);
}
