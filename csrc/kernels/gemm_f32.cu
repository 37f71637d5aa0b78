// True fp32 matrix product on the FMA pipes: the 32-bit mode of the serving path (no TF32, no bf16 splitting).
//
// 64 x 64 tiles, 256 threads, 4 x 4 outputs per thread, 16-deep shared-memory slices read through registers.  Any M, N, K
// and any row pitch: edges are guarded element by element.  The grouped form serves the expert layers of a routed
// feed-forward in one launch.
#include "gemm_f32.h"

#include "rb_common.cuh"

namespace rb {

constexpr int kSgTile = 64, kSgK = 16;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ a, long long lda, const float* __restrict__ b, long long ldb, float* __restrict__ d,
                long long ldd, int M, int N, int K, float alpha, const float* __restrict__ bias, int relu2, const int* __restrict__ tile_expert,
                const int* __restrict__ num_m_tiles, long long b_expert_stride) {
  __shared__ float as[kSgK][kSgTile + 4], bs[kSgK][kSgTile + 4];
  const int n0 = blockIdx.x * kSgTile;
  const int m0 = blockIdx.y * kSgTile;
  if (tile_expert) {
    if (m0 / 128 >= num_m_tiles[0]) return;
    const int e = tile_expert[m0 / 128];
    if (e < 0) return;
    b += static_cast<long long>(e) * b_expert_stride;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += kSgK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = i * 256 + threadIdx.x;
      const int r = idx >> 4, c = idx & 15;
      const bool kin = k0 + c < K;
      as[c][r] = (kin && m0 + r < M) ? a[static_cast<long long>(m0 + r) * lda + k0 + c] : 0.f;
      bs[c][r] = (kin && n0 + r < N) ? b[static_cast<long long>(n0 + r) * ldb + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSgK; ++k) {
      float av[4], bv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { av[i] = as[k][ty * 4 + i]; bv[i] = bs[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float v = alpha * acc[i][j] + (bias ? bias[n] : 0.f);
      if (relu2) { v = fmaxf(v, 0.f); v *= v; }
      d[static_cast<long long>(m) * ldd + n] = v;
    }
  }
}

}  // namespace rb

RB_API int rb_gemm_f32(const float* a, long long lda, const float* b, long long ldb, float* d, long long ldd, int M, int N,
                       int K, float alpha, const float* bias, int relu2, const int* tile_expert, const int* num_m_tiles, long long b_expert_stride,
                       void* stream_v) {
  if (M <= 0 || N <= 0 || K <= 0 || !a || !b || !d) return -1;
  if (tile_expert && (!num_m_tiles || b_expert_stride <= 0)) return -8;
  const dim3 grid((N + rb::kSgTile - 1) / rb::kSgTile, (M + rb::kSgTile - 1) / rb::kSgTile);
  if (grid.y > 65535) return -1;
  rb::gemm_f32_kernel<<<grid, 256, 0, reinterpret_cast<cudaStream_t>(stream_v)>>>(a, lda, b, ldb, d, ldd, M, N, K, alpha, bias, relu2,
                                                                                 tile_expert, num_m_tiles, b_expert_stride);
  return static_cast<int>(cudaGetLastError());
}
