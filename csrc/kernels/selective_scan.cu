// Mamba's selective scan: one step size per channel and token, one decay per channel and state number.
//
// LP lanes share a channel, each with NI of its state numbers in registers (fp32); CC = 128 / LP channels per CTA walk over the tokens of
// a segment.  Prompts: tiles of TT tokens, whose inputs are requested one tile ahead; step sizes (softplus) and dt x are formed once per
// channel and token in shared memory, the skip, the silu gate and the output scale are applied when the tile is stored.  The lanes'
// shares of y are summed for four tokens at a time, so that every step of the sum halves what is left.  One exponential per state number
// and token on the special-function unit is what the time goes to; the products run on packed pairs.  Decoded rows take a form without
// staging, whose traffic is the state, read and written once.
//
// fp32 operands take expf and plain arithmetic.
#include "recurrent.h"

#include "recurrent.cuh"

namespace rb {

constexpr int kSlThreads = 128;
constexpr float kSlLog2e = 1.4426950408889634f;

__device__ __forceinline__ float sl_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two fp32 numbers per instruction
__device__ __forceinline__ uint64_t sl_pack(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void sl_unpack(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t sl_fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t sl_mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// NI numbers of a channel's state.  `rate`: A, times log2(e) where the exponential is to base 2.
template <typename T, int NI> struct SlState;
template <int NI> struct SlState<float, NI> {
  float s[NI], rate[NI];
  static constexpr float kRate = 1.f;
  __device__ __forceinline__ void set(int i, float v, float r) { s[i] = v; rate[i] = r; }
  __device__ __forceinline__ float get(int i) const { return s[i]; }
  __device__ __forceinline__ float step(float dt, float u, const float* B, const float* C) {
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      s[i] = fmaf(expf(dt * rate[i]), s[i], u * B[i]);
      y = fmaf(s[i], C[i], y);
    }
    return y;
  }
};
template <int NI> struct SlState<__nv_bfloat16, NI> {
  uint64_t s[NI / 2], rate[NI / 2];
  static constexpr float kRate = kSlLog2e;
  __device__ __forceinline__ void set(int i, float v, float r) {
    float a, b, c, d;
    sl_unpack(s[i / 2], a, b);
    sl_unpack(rate[i / 2], c, d);
    s[i / 2] = i & 1 ? sl_pack(a, v) : sl_pack(v, b);
    rate[i / 2] = i & 1 ? sl_pack(c, r) : sl_pack(r, d);
  }
  __device__ __forceinline__ float get(int i) const {
    float a, b;
    sl_unpack(s[i / 2], a, b);
    return i & 1 ? b : a;
  }
  __device__ __forceinline__ float step(float dt, float u, const float* B, const float* C) {
    const uint64_t dt2 = sl_pack(dt, dt), u2 = sl_pack(u, u);
    uint64_t y2 = 0ull;
#pragma unroll
    for (int i = 0; i < NI / 2; ++i) {
      float lo, hi;
      sl_unpack(sl_mul2(dt2, rate[i]), lo, hi);
      s[i] = sl_fma2(sl_pack(sl_ex2(lo), sl_ex2(hi)), s[i], sl_mul2(u2, sl_pack(B[2 * i], B[2 * i + 1])));
      y2 = sl_fma2(s[i], sl_pack(C[2 * i], C[2 * i + 1]), y2);
    }
    float lo, hi;
    sl_unpack(y2, lo, hi);
    return lo + hi;
  }
};

// softplus of a step size: max(x, 0) + ln(1 + e), e = e^-|x|.  With bf16 operands ln(1 + e) = 2 atanh(e / (2 + e)) by the series of atanh,
// whose argument is at most 1/3 (relative error 2e-7).
template <typename T> __device__ __forceinline__ float sl_softplus(float x);
template <> __device__ __forceinline__ float sl_softplus<float>(float x) { return rc_softplus(x); }
template <> __device__ __forceinline__ float sl_softplus<__nv_bfloat16>(float x) {
  const float e = __expf(-fabsf(x)), s = __fdividef(e, 2.f + e), q = s * s;
  float p = fmaf(q, 1.f / 15.f, 1.f / 13.f);
  p = fmaf(p, q, 1.f / 11.f);
  p = fmaf(p, q, 1.f / 9.f);
  p = fmaf(p, q, 1.f / 7.f);
  p = fmaf(p, q, 1.f / 5.f);
  p = fmaf(p, q, 1.f / 3.f);
  return fmaxf(x, 0.f) + 2.f * s * fmaf(p, q, 1.f);
}

template <typename T, int NI>
__device__ __forceinline__ void sl_load_state(SlState<T, NI>& S, const RbSelectiveScanArgs& a, const RcSegment& s, int c, int n0, bool live) {
  const int n4 = (a.n + 3) & ~3;
  const float* st = a.state + (static_cast<long long>(s.slot) * a.inner + c) * n4;
  const float* A = a.A + static_cast<long long>(c) * a.n;
#pragma unroll
  for (int q = 0; q < NI; q += 4) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live && s.start > 0 && n0 + q < a.n) v = *reinterpret_cast<const float4*>(st + n0 + q);
    const float w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int n = n0 + q + i;
      S.set(q + i, n < a.n ? w[i] : 0.f, live && n < a.n ? A[n] * SlState<T, NI>::kRate : 0.f);
    }
  }
}
template <typename T, int NI>
__device__ __forceinline__ void sl_store_state(const SlState<T, NI>& S, const RbSelectiveScanArgs& a, const RcSegment& s, int c, int n0) {
  const int n4 = (a.n + 3) & ~3;
  float* st = a.state + (static_cast<long long>(s.slot) * a.inner + c) * n4;
#pragma unroll
  for (int q = 0; q < NI; q += 4)
    if (n0 + q < a.n) *reinterpret_cast<float4*>(st + n0 + q) = make_float4(S.get(q), S.get(q + 1), S.get(q + 2), S.get(q + 3));
}

template <typename T, int LP, int NI, int TT>
__global__ void __launch_bounds__(kSlThreads)
selective_scan_kernel(const RbSelectiveScanArgs a) {
  constexpr int CC = kSlThreads / LP, NP = LP * NI;
  constexpr int kItems = (TT * CC + kSlThreads - 1) / kSlThreads, kBC = (TT * NP + kSlThreads - 1) / kSlThreads;
  __shared__ __align__(16) float sB[TT][NP], sC[TT][NP];
  __shared__ float2 sIn[TT][CC];                     // step size, dt x
  __shared__ float sY[TT][CC];
  const int tid = threadIdx.x, p = tid % LP, cl = tid / LP, c0 = blockIdx.x * CC, c = c0 + cl, n0 = p * NI;
  const RcSegment s = rc_segment(a.segments, blockIdx.y, a.num_slots);
  if (s.len <= 0) return;
  const bool live = c < a.inner;
  SlState<T, NI> S;
  sl_load_state(S, a, s, c, n0, live);
  const T *X = reinterpret_cast<const T*>(a.x), *Z = reinterpret_cast<const T*>(a.z), *B = reinterpret_cast<const T*>(a.B),
          *C = reinterpret_cast<const T*>(a.C);
  // an item is one channel of one token of a tile: channel ic, tokens it0 + k * (kSlThreads / CC)
  const int ic = tid % CC, it0 = tid / CC;
  const bool item = c0 + ic < a.inner;
  const float bias = item ? a.dt_bias[c0 + ic] : 0.f, skip = item ? a.D[c0 + ic] : 0.f;
  float x[kItems], z[kItems], dt[kItems], nx[kItems], nz[kItems], b[kBC], cc[kBC];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int k = 0; k < kItems; ++k) {
      const int t = t0 + it0 + k * LP;
      nx[k] = nz[k] = dt[k] = 0.f;
      if (item && it0 + k * LP < TT && t < s.len) {
        const long long r = s.first + t;
        nx[k] = rc_get(X + r * a.ld_x + c0 + ic);
        nz[k] = rc_get(Z + r * a.ld_z + c0 + ic);
        dt[k] = a.dt_raw[r * a.ld_dt + c0 + ic];
      }
    }
#pragma unroll
    for (int k = 0; k < kBC; ++k) {
      const int i = tid + k * kSlThreads, t = t0 + i / NP, n = i % NP;
      b[k] = cc[k] = 0.f;
      if (i < TT * NP && t < s.len && n < a.n) {
        const long long r = s.first + t;
        b[k] = rc_get(B + r * a.ld_bc + n);
        cc[k] = rc_get(C + r * a.ld_bc + n);
      }
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < s.len; t0 += TT) {
#pragma unroll
    for (int k = 0; k < kItems; ++k) {
      x[k] = nx[k];
      z[k] = nz[k];
      // rows behind the end: a step of 0 leaves the state as it is
      const float d = t0 + it0 + k * LP < s.len ? sl_softplus<T>(dt[k] + bias) : 0.f;
      if (it0 + k * LP < TT) sIn[it0 + k * LP][ic] = make_float2(d, d * x[k]);
    }
#pragma unroll
    for (int k = 0; k < kBC; ++k) {
      const int i = tid + k * kSlThreads;
      if (i < TT * NP) { (&sB[0][0])[i] = b[k]; (&sC[0][0])[i] = cc[k]; }
    }
    __syncthreads();
    if (t0 + TT < s.len) fetch(t0 + TT);
#pragma unroll
    for (int t = 0; t < TT; t += 4) {
      float y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 in = sIn[t + k][cl];
        float vb[NI], vc[NI];
#pragma unroll
        for (int q = 0; q < NI; q += 4) {
          const float4 u = *reinterpret_cast<const float4*>(&sB[t + k][n0 + q]), w = *reinterpret_cast<const float4*>(&sC[t + k][n0 + q]);
          vb[q] = u.x; vb[q + 1] = u.y; vb[q + 2] = u.z; vb[q + 3] = u.w;
          vc[q] = w.x; vc[q + 1] = w.y; vc[q + 2] = w.z; vc[q + 3] = w.w;
        }
        y[k] = S.step(in.x, in.y, vb, vc);
      }
      if constexpr (LP == 1) {
#pragma unroll
        for (int k = 0; k < 4; ++k) sY[t + k][cl] = y[k];
      } else {
        const bool hi = p & 1;                       // this lane goes on with tokens 2, 3 instead of 0, 1
        float v0 = (hi ? y[2] : y[0]) + __shfl_xor_sync(0xffffffffu, hi ? y[0] : y[2], 1);
        float v1 = (hi ? y[3] : y[1]) + __shfl_xor_sync(0xffffffffu, hi ? y[1] : y[3], 1);
        if constexpr (LP == 2) {
          sY[t + 2 * hi][cl] = v0;
          sY[t + 2 * hi + 1][cl] = v1;
        } else {
          const bool odd = p & 2;                    // with the second of its two
          float v = (odd ? v1 : v0) + __shfl_xor_sync(0xffffffffu, odd ? v0 : v1, 2);
#pragma unroll
          for (int o = 4; o < LP; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
          if (p < 4) sY[t + 2 * hi + odd][cl] = v;
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kItems; ++k) {
      const int t = it0 + k * LP;
      if (item && t < TT && t0 + t < s.len)
        rc_put(reinterpret_cast<T*>(a.y) + (s.first + t0 + t) * a.ld_y + c0 + ic,
               a.scale * fmaf(skip, x[k], sY[t][ic]) * rc_silu<T>(z[k]));
    }
  }
  if (live) sl_store_state(S, a, s, c, n0);
}

// segments of one row
template <typename T, int LP, int NI>
__global__ void __launch_bounds__(kSlThreads)
selective_step_kernel(const RbSelectiveScanArgs a) {
  const int p = threadIdx.x % LP, c = blockIdx.x * (kSlThreads / LP) + threadIdx.x / LP, n0 = p * NI;
  const RcSegment s = rc_segment(a.segments, blockIdx.y, a.num_slots);
  if (s.len <= 0) return;
  const bool live = c < a.inner;                     // idle lanes stay for the shuffles
  const long long r = s.first;
  const float raw = live ? a.dt_raw[r * a.ld_dt + c] + a.dt_bias[c] : 0.f;
  const float x = live ? rc_get(reinterpret_cast<const T*>(a.x) + r * a.ld_x + c) : 0.f;
  const float z = live ? rc_get(reinterpret_cast<const T*>(a.z) + r * a.ld_z + c) : 0.f;
  float b[NI], cc[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const bool in = n0 + i < a.n;
    b[i] = in ? rc_get(reinterpret_cast<const T*>(a.B) + r * a.ld_bc + n0 + i) : 0.f;
    cc[i] = in ? rc_get(reinterpret_cast<const T*>(a.C) + r * a.ld_bc + n0 + i) : 0.f;
  }
  SlState<T, NI> S;
  sl_load_state(S, a, s, c, n0, live);
  const float dt = sl_softplus<T>(raw);
  float y = S.step(dt, dt * x, b, cc);
#pragma unroll
  for (int o = 1; o < LP; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (!live) return;
  sl_store_state(S, a, s, c, n0);
  if (p == 0) rc_put(reinterpret_cast<T*>(a.y) + r * a.ld_y + c, a.scale * fmaf(a.D[c], x, y) * rc_silu<T>(z));
}

template <typename T, int LP, int NI, int TT>
int sl_launch(const RbSelectiveScanArgs& a, cudaStream_t s) {
  constexpr int CC = kSlThreads / LP;
  const dim3 grid((a.inner + CC - 1) / CC, a.num_segments);
  if (a.single) selective_step_kernel<T, LP, NI><<<grid, kSlThreads, 0, s>>>(a);
  else selective_scan_kernel<T, LP, NI, TT><<<grid, kSlThreads, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int sl_pick(const RbSelectiveScanArgs& a, cudaStream_t s) {
  if (a.n <= 4) return sl_launch<T, 1, 4, 16>(a, s);
  if (a.n <= 8) return sl_launch<T, 2, 4, 16>(a, s);
  if (a.n <= 16) return sl_launch<T, 4, 4, 16>(a, s);
  if (a.n <= 32) return sl_launch<T, 8, 4, 16>(a, s);
  if (a.n <= 64) return sl_launch<T, 8, 8, 16>(a, s);
  if (a.n <= 128) return sl_launch<T, 16, 8, 16>(a, s);
  return sl_launch<T, 16, 16, 8>(a, s);
}

}  // namespace rb

RB_API int rb_selective_scan(const RbSelectiveScanArgs* args, void* stream_v) {
  const RbSelectiveScanArgs& a = *args;
  if (a.num_segments <= 0) return 0;
  if (!a.x || !a.z || !a.B || !a.C || !a.dt_raw || !a.dt_bias || !a.A || !a.D || !a.state || !a.y || !a.segments || a.inner <= 0 || a.n <= 0 ||
      a.n > 256 || a.num_slots <= 0 || a.num_segments > 65535)
    return -1;
  if (reinterpret_cast<uintptr_t>(a.state) & 15) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return a.f32 ? rb::sl_pick<float>(a, s) : rb::sl_pick<__nv_bfloat16>(a, s);
}
