// Gated delta rule.
//
// Scan form: one CTA owns 64 value columns of one head of one segment and keeps the state's columns in registers (fp32) while it
// walks over the tokens.  Per token one pass over the state gives both S^T k and S^T q of the state before the token; the read-out
// after the write follows as decay S^T q + (k . q) u, so a token costs one reduction over the CTA.  With segments of one token
// this is the decode step.  It takes bf16 and fp32 and any sizes up to 256 state rows.
#include "recurrent.h"

#include "recurrent.cuh"

namespace rb {

constexpr int kDrTile = 8;                 // tokens staged at a time
constexpr int kDrCols = 64;                // value columns of a CTA
constexpr float kDrUnitEps = 1e-6f;

template <typename T, int NI>              // state rows per thread: dk <= 8 NI
__global__ void __launch_bounds__(128)
delta_rule_scan_kernel(const RbDeltaRuleArgs a) {
  __shared__ float sQ[kDrTile][8 * NI], sK[kDrTile][8 * NI];
  __shared__ __align__(16) float sV[kDrTile][kDrCols];
  __shared__ __align__(16) float red[2][2][4][kDrCols];      // [parity][S^T k, S^T q][warp][column]
  __shared__ float sBeta[kDrTile], sDecay[kDrTile], sKQ[kDrTile];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c4 = tid & 15, ng = tid >> 4;
  const int c0 = blockIdx.x * kDrCols, h = blockIdx.y;
  const RcSegment s = rc_segment(a.segments, blockIdx.z, a.num_slots);
  if (s.len <= 0) return;
  const int v4 = (a.dv + 3) & ~3;
  const int col = c0 + c4 * 4;
  const bool live = col < v4;
  const int g = h / (a.heads / a.kv_heads);
  float4* st = reinterpret_cast<float4*>(a.state + (static_cast<long long>(s.slot) * a.heads + h) * a.dk * v4 + col);
  const int row4 = v4 / 4;
  float4 S[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = ng + 8 * i;
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live && s.start > 0 && n < a.dk) S[i] = st[n * row4];
  }
  const float rate = expf(a.a_log[h]), dt_bias = a.dt_bias[h], qscale = rsqrtf(static_cast<float>(a.dk));
  const T* qkv = reinterpret_cast<const T*>(a.qkv);
  const long long offQ = static_cast<long long>(g) * a.dk, offK = static_cast<long long>(a.kv_heads + g) * a.dk;
  const long long offV = 2ll * a.kv_heads * a.dk + static_cast<long long>(h) * a.dv + c0;
  for (int t0 = 0; t0 < s.len; t0 += kDrTile) {
    const int m = min(kDrTile, s.len - t0);
    for (int i = tid; i < m * 8 * NI; i += 128) {
      const int t = i / (8 * NI), n = i - t * (8 * NI);
      const T* row = qkv + (s.first + t0 + t) * a.ld_qkv;
      sQ[t][n] = n < a.dk ? rc_get(row + offQ + n) : 0.f;
      sK[t][n] = n < a.dk ? rc_get(row + offK + n) : 0.f;
    }
    for (int i = tid; i < m * kDrCols; i += 128) {
      const int t = i / kDrCols, c = i - t * kDrCols;
      sV[t][c] = c0 + c < a.dv ? rc_get(qkv + (s.first + t0 + t) * a.ld_qkv + offV + c) : 0.f;
    }
    if (tid < m) {
      const long long at = (s.first + t0 + tid) * a.ld_ab + h;
      sBeta[tid] = rc_sigmoid(a.b_raw[at]);
      sDecay[tid] = expf(-rate * rc_softplus(a.a_raw[at] + dt_bias));
    }
    __syncthreads();
    // unit vectors: a warp takes two tokens
    for (int t = 2 * warp; t < min(m, 2 * warp + 2); ++t) {
      float qq = 0.f, kk = 0.f;
      for (int n = lane; n < 8 * NI; n += 32) { qq = fmaf(sQ[t][n], sQ[t][n], qq); kk = fmaf(sK[t][n], sK[t][n], kk); }
      const float rq = qscale / sqrtf(warp_sum(qq) + kDrUnitEps), rk = 1.f / sqrtf(warp_sum(kk) + kDrUnitEps);
      float kq = 0.f;
      for (int n = lane; n < 8 * NI; n += 32) {
        const float q = sQ[t][n] * rq, k = sK[t][n] * rk;
        sQ[t][n] = q;
        sK[t][n] = k;
        kq = fmaf(q, k, kq);
      }
      kq = warp_sum(kq);
      if (lane == 0) sKQ[t] = kq;
    }
    __syncthreads();
    for (int t = 0; t < m; ++t) {
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f), z = y;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float k = sK[t][ng + 8 * i], q = sQ[t][ng + 8 * i];
        y.x = fmaf(k, S[i].x, y.x); y.y = fmaf(k, S[i].y, y.y); y.z = fmaf(k, S[i].z, y.z); y.w = fmaf(k, S[i].w, y.w);
        z.x = fmaf(q, S[i].x, z.x); z.y = fmaf(q, S[i].y, z.y); z.z = fmaf(q, S[i].z, z.z); z.w = fmaf(q, S[i].w, z.w);
      }
      y.x += __shfl_xor_sync(0xffffffffu, y.x, 16); y.y += __shfl_xor_sync(0xffffffffu, y.y, 16);
      y.z += __shfl_xor_sync(0xffffffffu, y.z, 16); y.w += __shfl_xor_sync(0xffffffffu, y.w, 16);
      z.x += __shfl_xor_sync(0xffffffffu, z.x, 16); z.y += __shfl_xor_sync(0xffffffffu, z.y, 16);
      z.z += __shfl_xor_sync(0xffffffffu, z.z, 16); z.w += __shfl_xor_sync(0xffffffffu, z.w, 16);
      const int par = t & 1;
      if (lane < 16) {
        *reinterpret_cast<float4*>(&red[par][0][warp][c4 * 4]) = y;
        *reinterpret_cast<float4*>(&red[par][1][warp][c4 * 4]) = z;
      }
      __syncthreads();
      float sk[4] = {0.f, 0.f, 0.f, 0.f}, sq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float4 u = *reinterpret_cast<const float4*>(&red[par][0][w][c4 * 4]);
        const float4 v = *reinterpret_cast<const float4*>(&red[par][1][w][c4 * 4]);
        sk[0] += u.x; sk[1] += u.y; sk[2] += u.z; sk[3] += u.w;
        sq[0] += v.x; sq[1] += v.y; sq[2] += v.z; sq[3] += v.w;
      }
      const float da = sDecay[t], beta = sBeta[t], kq = sKQ[t];
      float u[4], o[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        u[j] = beta * (sV[t][c4 * 4 + j] - da * sk[j]);
        o[j] = fmaf(da, sq[j], kq * u[j]);
      }
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float k = sK[t][ng + 8 * i];
        S[i].x = fmaf(da, S[i].x, k * u[0]); S[i].y = fmaf(da, S[i].y, k * u[1]);
        S[i].z = fmaf(da, S[i].z, k * u[2]); S[i].w = fmaf(da, S[i].w, k * u[3]);
      }
      if (ng == 0) {
        T* out = reinterpret_cast<T*>(a.o) + (s.first + t0 + t) * a.ld_o + static_cast<long long>(h) * a.dv;
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (col + j < a.dv) rc_put(out + col + j, o[j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = ng + 8 * i;
    if (live && n < a.dk) st[n * row4] = S[i];
  }
}

template <typename T>
int dr_launch(const RbDeltaRuleArgs& a, cudaStream_t s) {
  const dim3 grid((a.dv + kDrCols - 1) / kDrCols, a.heads, a.num_segments);
  if (a.dk <= 32) delta_rule_scan_kernel<T, 4><<<grid, 128, 0, s>>>(a);
  else if (a.dk <= 64) delta_rule_scan_kernel<T, 8><<<grid, 128, 0, s>>>(a);
  else if (a.dk <= 128) delta_rule_scan_kernel<T, 16><<<grid, 128, 0, s>>>(a);
  else delta_rule_scan_kernel<T, 32><<<grid, 128, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace rb

RB_API int rb_delta_rule_scan(const RbDeltaRuleArgs* args, void* stream_v) {
  const RbDeltaRuleArgs& a = *args;
  if (a.num_segments <= 0) return 0;
  if (!a.qkv || !a.a_raw || !a.b_raw || !a.dt_bias || !a.a_log || !a.state || !a.o || !a.segments || a.heads <= 0 ||
      a.kv_heads <= 0 || a.heads % a.kv_heads || a.dk <= 0 || a.dk > 256 || a.dv <= 0 || a.num_slots <= 0 ||
      a.num_segments > 65535 || a.heads > 65535)
    return -1;
  if (reinterpret_cast<uintptr_t>(a.state) & 15) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return a.f32 ? rb::dr_launch<float>(a, s) : rb::dr_launch<__nv_bfloat16>(a, s);
}
