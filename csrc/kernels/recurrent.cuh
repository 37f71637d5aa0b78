// Device helpers of the recurrent layers.
#pragma once
#include "rb_common.cuh"

namespace rb {

struct RcSegment {
  int first, len, slot, start;
};
// Row `i` of the segment table.  A slot outside the state tensor counts as an empty segment.
__device__ __forceinline__ RcSegment rc_segment(const int* table, int i, int num_slots) {
  const int4 u = reinterpret_cast<const int4*>(table)[i];
  RcSegment s = {u.x, u.y, u.z, u.w};
  if (s.slot < 0 || s.slot >= num_slots) s.len = 0;
  return s;
}

__device__ __forceinline__ float rc_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float rc_get(const float* p) { return *p; }
__device__ __forceinline__ void rc_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void rc_put(float* p, float v) { *p = v; }

__device__ __forceinline__ float rc_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float rc_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// N consecutive elements as fp32
template <typename T, int N> struct RcVec;
template <typename T> struct RcVec<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = rc_get(p); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { rc_put(p, v[0]); }
};
template <> struct RcVec<__nv_bfloat16, 8> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = unpack_bf16x2(w[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]),
                                              pack_bf16x2(v[6], v[7]));
  }
};
template <> struct RcVec<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  }
};
template <> struct RcVec<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};

// silu for a result that is rounded to T: full precision in 32-bit
template <typename T> __device__ __forceinline__ float rc_silu(float x);
template <> __device__ __forceinline__ float rc_silu<float>(float x) { return x / (1.f + expf(-x)); }
template <> __device__ __forceinline__ float rc_silu<__nv_bfloat16>(float x) { return silu(x); }

}  // namespace rb
