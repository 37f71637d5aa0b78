// What the two decode kernels of latent attention share.
#pragma once
#include "latent_attention.h"

#include "rb_common.cuh"

namespace rb {

// Tokens per slice when a context is cut into `splits`: whole tiles of 128.
__host__ __device__ __forceinline__ int latent_chunk(int ctx, int splits) {
  return ((ctx + splits - 1) / splits + 127) / 128 * 128;
}

// The tensor-core form (latent_decode_tc.cu); -9: a problem it does not take.
int latent_decode_tc(const RbLatentDecodeArgs& a, int splits, cudaStream_t s);

}  // namespace rb
