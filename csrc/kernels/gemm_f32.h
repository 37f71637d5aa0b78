// C interface of the true fp32 matrix product (gemm_f32.cu).  All pointers are device pointers.
#pragma once
#ifdef __cplusplus
extern "C" {
#endif
// d[M, N] = act(alpha * a[M, K] b[N, K]^T + bias), bias fp32 [N] or NULL, act: the square of relu with relu2; all fp32, products and sums in fp32 FMA (no reduced-precision tensor-core mode).
// Grouped form (tile_expert != NULL): rows of a / d are grouped by expert in 128-row tiles (moe.h), tile i uses
// b + tile_expert[i] * b_expert_stride; num_m_tiles [1] is the number of live tiles.
int rb_gemm_f32(const float* a, long long lda, const float* b, long long ldb, float* d, long long ldd, int M, int N, int K,
                float alpha, const float* bias, int relu2, const int* tile_expert, const int* num_m_tiles, long long b_expert_stride,
                void* stream);
#ifdef __cplusplus
}
#endif
