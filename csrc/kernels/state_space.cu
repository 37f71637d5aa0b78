// Mamba-2 state-space recurrence, and the same with one fixed decay per head (retention).
//
// Scan form: one CTA owns 64 value columns of one head of one segment and keeps the state's columns in registers (fp32) while it
// walks over the tokens; B, C, x and the step sizes of 8 tokens at a time are staged in shared memory.  With segments of one
// token this is the decode step: the state is read and written once, which is all the traffic that matters.  It takes bf16 and
// fp32 and any sizes up to 256 state rows.
#include "recurrent.h"

#include "recurrent.cuh"

namespace rb {

constexpr int kSsTile = 8;                 // tokens staged at a time
constexpr int kSsCols = 64;                // value columns of a CTA

template <typename T, int NI>              // state rows per thread: n <= 8 NI
__global__ void __launch_bounds__(128)
state_space_scan_kernel(const RbStateSpaceArgs a) {
  __shared__ float sB[kSsTile][8 * NI], sC[kSsTile][8 * NI];
  __shared__ __align__(16) float sX[kSsTile][kSsCols];
  __shared__ __align__(16) float sY[kSsTile][4][kSsCols];
  __shared__ float sDt[kSsTile], sDecay[kSsTile];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c4 = tid & 15, ng = tid >> 4;
  const int c0 = blockIdx.x * kSsCols, h = blockIdx.y;
  const RcSegment s = rc_segment(a.segments, blockIdx.z, a.num_slots);
  if (s.len <= 0) return;
  const int p4 = (a.p + 3) & ~3;
  const int col = c0 + c4 * 4;
  const bool live = col < p4;
  const int g = h / (a.heads / a.groups);
  float4* st = reinterpret_cast<float4*>(a.state + (static_cast<long long>(s.slot) * a.heads + h) * a.n * p4 + col);
  const int row4 = p4 / 4;                 // float4 pitch of the state
  float4 S[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = ng + 8 * i;
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live && s.start > 0 && n < a.n) S[i] = st[n * row4];
  }
  const bool fixed = a.decay != nullptr;
  const float rate = fixed ? 0.f : expf(a.a_log[h]), dt_bias = fixed ? 0.f : a.dt_bias[h], dskip = a.D ? a.D[h] : 0.f;
  const T* xbc = reinterpret_cast<const T*>(a.xbc);
  const long long offB = static_cast<long long>(a.heads) * a.p + static_cast<long long>(g) * a.n;
  const long long offC = offB + static_cast<long long>(a.groups) * a.n;
  for (int t0 = 0; t0 < s.len; t0 += kSsTile) {
    const int m = min(kSsTile, s.len - t0);
    for (int i = tid; i < m * 8 * NI; i += 128) {
      const int t = i / (8 * NI), n = i - t * (8 * NI);
      const T* row = xbc + (s.first + t0 + t) * a.ld_xbc;
      sB[t][n] = n < a.n ? rc_get(row + offB + n) : 0.f;
      sC[t][n] = n < a.n ? rc_get(row + offC + n) : 0.f;
    }
    for (int i = tid; i < m * kSsCols; i += 128) {
      const int t = i / kSsCols, c = i - t * kSsCols;
      sX[t][c] = c0 + c < a.p ? rc_get(xbc + (s.first + t0 + t) * a.ld_xbc + static_cast<long long>(h) * a.p + c0 + c) : 0.f;
    }
    if (tid < m) {
      const float dt = fixed ? 1.f : rc_softplus(a.dt_raw[(s.first + t0 + tid) * a.ld_dt + h] + dt_bias);
      sDt[tid] = dt;
      sDecay[tid] = fixed ? a.decay[h] : expf(-rate * dt);
    }
    __syncthreads();
    for (int t = 0; t < m; ++t) {
      const float4 x = *reinterpret_cast<const float4*>(&sX[t][c4 * 4]);
      const float dt = sDt[t], da = sDecay[t];
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float b = sB[t][ng + 8 * i] * dt, c = sC[t][ng + 8 * i];
        S[i].x = fmaf(da, S[i].x, b * x.x); S[i].y = fmaf(da, S[i].y, b * x.y);
        S[i].z = fmaf(da, S[i].z, b * x.z); S[i].w = fmaf(da, S[i].w, b * x.w);
        y.x = fmaf(c, S[i].x, y.x); y.y = fmaf(c, S[i].y, y.y); y.z = fmaf(c, S[i].z, y.z); y.w = fmaf(c, S[i].w, y.w);
      }
      y.x += __shfl_xor_sync(0xffffffffu, y.x, 16); y.y += __shfl_xor_sync(0xffffffffu, y.y, 16);
      y.z += __shfl_xor_sync(0xffffffffu, y.z, 16); y.w += __shfl_xor_sync(0xffffffffu, y.w, 16);
      if (lane < 16) *reinterpret_cast<float4*>(&sY[t][warp][c4 * 4]) = y;
    }
    __syncthreads();
    for (int i = tid; i < m * kSsCols; i += 128) {
      const int t = i / kSsCols, c = i - t * kSsCols;
      if (c0 + c >= a.p) continue;
      const float v = (sY[t][0][c] + sY[t][1][c]) + (sY[t][2][c] + sY[t][3][c]) + dskip * sX[t][c];
      rc_put(reinterpret_cast<T*>(a.y) + (s.first + t0 + t) * a.ld_y + static_cast<long long>(h) * a.p + c0 + c, v);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = ng + 8 * i;
    if (live && n < a.n) st[n * row4] = S[i];
  }
}

template <typename T>
int ss_launch(const RbStateSpaceArgs& a, cudaStream_t s) {
  const dim3 grid((a.p + kSsCols - 1) / kSsCols, a.heads, a.num_segments);
  if (a.n <= 32) state_space_scan_kernel<T, 4><<<grid, 128, 0, s>>>(a);
  else if (a.n <= 64) state_space_scan_kernel<T, 8><<<grid, 128, 0, s>>>(a);
  else if (a.n <= 128) state_space_scan_kernel<T, 16><<<grid, 128, 0, s>>>(a);
  else state_space_scan_kernel<T, 32><<<grid, 128, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace rb

RB_API int rb_state_space_scan(const RbStateSpaceArgs* args, void* stream_v) {
  const RbStateSpaceArgs& a = *args;
  if (a.num_segments <= 0) return 0;
  if (!a.xbc || (!a.decay && (!a.dt_raw || !a.dt_bias || !a.a_log)) || !a.state || !a.y || !a.segments || a.heads <= 0 || a.groups <= 0 ||
      a.heads % a.groups || a.p <= 0 || a.n <= 0 || a.n > 256 || a.num_slots <= 0 || a.num_segments > 65535 || a.heads > 65535)
    return -1;
  if (reinterpret_cast<uintptr_t>(a.state) & 15) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return a.f32 ? rb::ss_launch<float>(a, s) : rb::ss_launch<__nv_bfloat16>(a, s);
}
