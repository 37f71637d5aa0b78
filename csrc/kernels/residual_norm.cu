// Norm on a sublayer's output, added to a 32-bit residual stream, in one pass: x += norm(source), h = copy of x for the
// next matrix product.  The source is a plain row (attention output projection) or the weighted sum of a token's expert
// rows plus the shared expert's row, so a routed feed-forward's combine, norm and residual add are one launch.
// Where a norm stands in front of the next sublayer too, h is that norm of the new residual.
// Statistics, sums and the residual are fp32; one CTA owns a row and keeps it in registers.
//
// The second kernel serves blocks whose sublayers are computed side by side: up to two RMS-normed outputs and a plain one are
// added to the residual, and the dynamic tanh in front of the next block is taken on the way.
#include "residual_norm.h"

#include "rb_common.cuh"

namespace rb {

template <int VEC>
__device__ __forceinline__ void rn_load(const void* base, long long off, int f32, float (&v)[VEC]) {
  if (VEC == 4) {
    if (f32) {
      const float4 u = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(base) + off);
      v[0] = u.x; v[1 % VEC] = u.y; v[2 % VEC] = u.z; v[3 % VEC] = u.w;
    } else {
      const uint2 u = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(base) + off);
      const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
      v[0] = a.x; v[1 % VEC] = a.y; v[2 % VEC] = b.x; v[3 % VEC] = b.y;
    }
  } else {
    v[0] = f32 ? reinterpret_cast<const float*>(base)[off]
               : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(base)[off]);
  }
}
template <int VEC>
__device__ __forceinline__ void rn_store(void* base, long long off, int f32, const float (&v)[VEC]) {
  if (VEC == 4) {
    if (f32)
      *reinterpret_cast<float4*>(reinterpret_cast<float*>(base) + off) = make_float4(v[0], v[1 % VEC], v[2 % VEC], v[3 % VEC]);
    else
      *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(base) + off) =
          make_uint2(pack_bf16x2(v[0], v[1 % VEC]), pack_bf16x2(v[2 % VEC], v[3 % VEC]));
  } else if (f32) {
    reinterpret_cast<float*>(base)[off] = v[0];
  } else {
    reinterpret_cast<__nv_bfloat16*>(base)[off] = __float2bfloat16(v[0]);
  }
}

// sum over the CTA; `red` holds one float per warp
__device__ __forceinline__ float rn_block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warps = blockDim.x >> 5;
  if (warps == 1) return v;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < warps; ++i) s += red[i];
  return s;
}

template <int VEC, int CH>
__global__ void __launch_bounds__(256)
residual_norm_kernel(const RbResidualNormArgs a) {
  __shared__ float red[8];
  const int t = blockIdx.x, n = a.n;
  float v[CH][VEC], xr[CH][VEC];
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int col = (c * blockDim.x + threadIdx.x) * VEC;
#pragma unroll
    for (int i = 0; i < VEC; ++i) { v[c][i] = 0.f; xr[c][i] = 0.f; }
    if (col >= n) continue;
    if (a.x) rn_load<VEC>(a.x, t * a.ldx + col, 1, xr[c]);
    if (a.add) rn_load<VEC>(a.add, t * a.ld_add + col, a.y_f32, v[c]);
    if (a.slot_pos) {
      for (int j = 0; j < a.k; ++j) {                     // fixed order: reproducible
        const float w = a.slot_w ? a.slot_w[static_cast<long long>(t) * a.k + j] : 1.f;
        float u[VEC];
        rn_load<VEC>(a.y, a.slot_pos[static_cast<long long>(t) * a.k + j] * a.ldy + col, a.y_f32, u);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[c][i] = fmaf(w, u[i], v[c][i]);
      }
    } else {
      float u[VEC];
      rn_load<VEC>(a.y, t * a.ldy + col, a.y_f32, u);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[c][i] += u[i];
    }
  }
  const float inv_n = 1.f / static_cast<float>(n);
  const bool plain = a.gamma == nullptr;             // the source is added as it is
  float mean = 0.f;
  if (!a.rms && !plain) {
    float s = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c)
#pragma unroll
      for (int i = 0; i < VEC; ++i) s += v[c][i];
    mean = rn_block_sum(s, red) * inv_n;
  }
  float rstd = 1.f;
  if (!plain) {
    float sq = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c)
      if ((c * blockDim.x + threadIdx.x) * VEC < n) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) { const float d = v[c][i] - mean; sq += d * d; }
      }
    rstd = rsqrtf(rn_block_sum(sq, red) * inv_n + a.eps);
  }
  float next = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int col = (c * blockDim.x + threadIdx.x) * VEC;
    if (col >= n) continue;
    float g[VEC], b[VEC], o[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) { g[i] = 1.f; b[i] = 0.f; }
    if (!plain) rn_load<VEC>(a.gamma, col, a.param_f32, g);
    if (a.beta) rn_load<VEC>(a.beta, col, a.param_f32, b);
#pragma unroll
    for (int i = 0; i < VEC; ++i) o[i] = xr[c][i] + ((v[c][i] - mean) * rstd * g[i] + b[i]);
    if (a.x) rn_store<VEC>(a.x, t * a.ldx + col, 1, o);
    if (a.next_gamma) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) { xr[c][i] = o[i]; next = fmaf(o[i], o[i], next); }
    } else if (a.h) {
      rn_store<VEC>(a.h, t * a.ldh + col, a.h_f32, o);
    }
  }
  if (!a.next_gamma) return;
  const float scale = 1.f / sqrtf(rn_block_sum(next, red) * inv_n + a.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int col = (c * blockDim.x + threadIdx.x) * VEC;
    if (col >= n) continue;
    float g[VEC];
    rn_load<VEC>(a.next_gamma, col, a.param_f32, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) g[i] *= xr[c][i] * scale;
    rn_store<VEC>(a.h, t * a.ldh + col, a.h_f32, g);
  }
}

template <int VEC>
int rn_launch(const RbResidualNormArgs& a, cudaStream_t s) {
  const int units = (a.n + VEC - 1) / VEC;
  const int threads = units <= 64 ? 64 : units <= 128 ? 128 : 256;
  const int ch = (units + threads - 1) / threads;
  if (ch <= 1) residual_norm_kernel<VEC, 1><<<a.rows, threads, 0, s>>>(a);
  else if (ch <= 2) residual_norm_kernel<VEC, 2><<<a.rows, threads, 0, s>>>(a);
  else if (ch <= 4) residual_norm_kernel<VEC, 4><<<a.rows, threads, 0, s>>>(a);
  else if (ch <= 8) residual_norm_kernel<VEC, 8><<<a.rows, threads, 0, s>>>(a);
  else if (ch <= 16) residual_norm_kernel<VEC, 16><<<a.rows, threads, 0, s>>>(a);
  else return -6;
  return static_cast<int>(cudaGetLastError());
}

// two sums over the CTA at once; `red` holds two floats per warp
__device__ __forceinline__ float2 rn_block_sum2(float v, float w, float2* red) {
  v = warp_sum(v);
  w = warp_sum(w);
  const int warps = blockDim.x >> 5;
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(v, w);
  __syncthreads();
  float2 s = make_float2(0.f, 0.f);
  for (int i = 0; i < warps; ++i) { s.x += red[i].x; s.y += red[i].y; }
  return s;
}

template <int VEC, int CH>
__global__ void __launch_bounds__(256)
stream_update_kernel(const RbStreamUpdateArgs a) {
  __shared__ float2 red[8];
  const int t = blockIdx.x, n = a.n;
  float x[CH][VEC], va[CH][VEC], vb[CH][VEC], v[CH][VEC];
  float sa = 0.f, sb = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int col = (c * blockDim.x + threadIdx.x) * VEC;
#pragma unroll
    for (int i = 0; i < VEC; ++i) { x[c][i] = 0.f; va[c][i] = 0.f; vb[c][i] = 0.f; v[c][i] = 0.f; }
    if (col >= n) continue;
    rn_load<VEC>(a.x, t * a.ldx + col, 1, x[c]);
    if (a.a) rn_load<VEC>(a.a, t * a.lda + col, a.y_f32, va[c]);
    if (a.b) rn_load<VEC>(a.b, t * a.ldb + col, a.y_f32, vb[c]);
    if (a.c) rn_load<VEC>(a.c, t * a.ldc + col, a.y_f32, v[c]);
#pragma unroll
    for (int i = 0; i < VEC; ++i) { sa = fmaf(va[c][i], va[c][i], sa); sb = fmaf(vb[c][i], vb[c][i], sb); }
  }
  const float inv_n = 1.f / static_cast<float>(n);
  float ra = 0.f, rb_ = 0.f;
  if (a.a || a.b) {
    const float2 sums = rn_block_sum2(sa, sb, red);
    ra = a.normed / sqrtf(sums.x * inv_n + a.eps);
    rb_ = a.normed / sqrtf(sums.y * inv_n + a.eps);
  }
  const bool add = a.a || a.b || a.c;
  const float alpha = a.h ? a.alpha[0] : 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int col = (c * blockDim.x + threadIdx.x) * VEC;
    if (col >= n) continue;
    float w[VEC];
    if (a.a) {
      rn_load<VEC>(a.wa, col, 1, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[c][i] = fmaf(va[c][i] * ra, w[i], v[c][i]);
    }
    if (a.b) {
      rn_load<VEC>(a.wb, col, 1, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[c][i] = fmaf(vb[c][i] * rb_, w[i], v[c][i]);
    }
    if (add) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[c][i] = fmaf(a.mult, v[c][i], x[c][i]);
      rn_store<VEC>(a.x, t * a.ldx + col, 1, x[c]);
    }
    if (a.h) {
      float b[VEC], o[VEC];
      rn_load<VEC>(a.gamma, col, 1, w);
      rn_load<VEC>(a.beta, col, 1, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = fmaf(tanhf(alpha * x[c][i]), w[i], b[i]);
      rn_store<VEC>(a.h, t * a.ldh + col, a.h_f32, o);
    }
  }
}

template <int VEC>
int su_launch(const RbStreamUpdateArgs& a, cudaStream_t s) {
  const int units = (a.n + VEC - 1) / VEC;
  const int threads = units <= 64 ? 64 : units <= 128 ? 128 : 256;
  const int ch = (units + threads - 1) / threads;
  if (ch <= 1) stream_update_kernel<VEC, 1><<<a.rows, threads, 0, s>>>(a);
  else if (ch <= 2) stream_update_kernel<VEC, 2><<<a.rows, threads, 0, s>>>(a);
  else if (ch <= 4) stream_update_kernel<VEC, 4><<<a.rows, threads, 0, s>>>(a);
  else if (ch <= 8) stream_update_kernel<VEC, 8><<<a.rows, threads, 0, s>>>(a);
  else if (ch <= 16) stream_update_kernel<VEC, 16><<<a.rows, threads, 0, s>>>(a);
  else return -6;
  return static_cast<int>(cudaGetLastError());
}

}  // namespace rb

RB_API int rb_stream_update(const RbStreamUpdateArgs* args, void* stream_v) {
  const RbStreamUpdateArgs& a = *args;
  if (a.rows <= 0) return 0;
  if (a.n <= 0 || !a.x || (a.a && !a.wa) || (a.b && !a.wb) || (a.h && (!a.alpha || !a.gamma || !a.beta))) return -1;
  const void* ptrs[9] = {a.a, a.b, a.c, a.wa, a.wb, a.x, a.gamma, a.beta, a.h};
  uintptr_t bits = 0;
  for (int i = 0; i < 9; ++i) bits |= reinterpret_cast<uintptr_t>(ptrs[i]);
  const bool vec = !(bits & 15) && !((a.n | a.lda | a.ldb | a.ldc | a.ldx | a.ldh) & 3);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return vec ? rb::su_launch<4>(a, s) : rb::su_launch<1>(a, s);
}

RB_API int rb_residual_norm(const RbResidualNormArgs* args, void* stream_v) {
  const RbResidualNormArgs& a = *args;
  if (a.rows <= 0 || a.n <= 0 || !a.y || (!a.gamma && (!a.x || a.beta)) || (!a.x && !a.h)) return -1;
  if (a.slot_pos && a.k <= 0) return -1;
  if (a.next_gamma && (!a.x || !a.h)) return -1;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.add) |
                         reinterpret_cast<uintptr_t>(a.gamma) | reinterpret_cast<uintptr_t>(a.beta) |
                         reinterpret_cast<uintptr_t>(a.next_gamma) | reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.h);
  const bool vec = !(bits & 15) && !((a.n | a.ldy | a.ld_add | a.ldx | a.ldh) & 3);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return vec ? rb::rn_launch<4>(a, s) : rb::rn_launch<1>(a, s);
}
