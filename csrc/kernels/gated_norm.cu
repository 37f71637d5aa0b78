// RMS norm over equal parts of a row with a silu gate before or behind it: the output stage of the recurrent mixers.  Between
// 8 lanes and a CTA own one part, by its size, and keep it in registers; sums are fp32.
#include "recurrent.h"

#include "recurrent.cuh"

namespace rb {

// sum over the lanes that own a part: up to a warp, or the whole CTA
template <int L>
__device__ __forceinline__ float gn_sum(float v, float* red) {
#pragma unroll
  for (int o = (L < 32 ? L : 32) / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if (L <= 32) return v;
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < L / 32; ++i) s += red[i];
  return s;
}

template <typename T, int VEC, int CH, int L>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const RbGatedNormArgs a) {
  __shared__ float red[8];
  const int sub = L <= 32 ? threadIdx.x & (L - 1) : threadIdx.x;
  const long long total = static_cast<long long>(a.rows) * a.parts;
  long long item = L <= 32 ? static_cast<long long>(blockIdx.x) * (256 / (L < 32 ? L : 32)) + threadIdx.x / L : blockIdx.x;
  const bool idle = item >= total;                 // the last CTA's: they stay for the shuffles and compute a part once more
  if (idle) item = total - 1;
  const long long t = item / a.parts;
  const int part = static_cast<int>(item - t * a.parts);
  const long long base = static_cast<long long>(part) * a.part_n;
  const T* y = reinterpret_cast<const T*>(a.y) + t * a.ld_y + base;
  const T* z = reinterpret_cast<const T*>(a.z) + t * a.ld_z + base;
  T* out = reinterpret_cast<T*>(a.out) + t * a.ld_o + base;
  const float* w = a.weight ? a.weight + (a.weight_n == a.part_n ? 0 : base) : nullptr;
  float u[CH][VEC], gate[CH][VEC];
  float sq = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int col = (c * L + sub) * VEC;
    if (col >= a.part_n) continue;
    RcVec<T, VEC>::load(y + col, u[c]);
    RcVec<T, VEC>::load(z + col, gate[c]);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      gate[c][i] = rc_silu<T>(gate[c][i]);
      if (a.gate_first) u[c][i] *= gate[c][i];
      sq = fmaf(u[c][i], u[c][i], sq);
    }
  }
  const float r = 1.f / sqrtf(gn_sum<L>(sq, red) / static_cast<float>(a.part_n) + a.eps);
  if (idle) return;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int col = (c * L + sub) * VEC;
    if (col >= a.part_n) continue;
    float o[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) o[i] = u[c][i] * r * (w ? w[col + i] : 1.f) * (a.gate_first ? 1.f : gate[c][i]);
    RcVec<T, VEC>::store(out + col, o);
  }
}

// any size and alignment: the part is read twice
template <typename T>
__global__ void __launch_bounds__(256)
gated_norm_any_kernel(const RbGatedNormArgs a) {
  __shared__ float red[8];
  const long long t = blockIdx.x / a.parts;
  const int part = blockIdx.x % a.parts;
  const long long base = static_cast<long long>(part) * a.part_n;
  const T* y = reinterpret_cast<const T*>(a.y) + t * a.ld_y + base;
  const T* z = reinterpret_cast<const T*>(a.z) + t * a.ld_z + base;
  const float* w = a.weight ? a.weight + (a.weight_n == a.part_n ? 0 : base) : nullptr;
  float sq = 0.f;
  for (int c = threadIdx.x; c < a.part_n; c += 256) {
    const float u = rc_get(y + c) * (a.gate_first ? rc_silu<T>(rc_get(z + c)) : 1.f);
    sq = fmaf(u, u, sq);
  }
  const float r = 1.f / sqrtf(gn_sum<256>(sq, red) / static_cast<float>(a.part_n) + a.eps);
  for (int c = threadIdx.x; c < a.part_n; c += 256)
    rc_put(reinterpret_cast<T*>(a.out) + t * a.ld_o + base + c, rc_get(y + c) * rc_silu<T>(rc_get(z + c)) * r * (w ? w[c] : 1.f));
}

template <typename T, int VEC, int L>
int gn_launch(const RbGatedNormArgs& a, cudaStream_t s) {
  const long long items = static_cast<long long>(a.rows) * a.parts;
  const int per = L <= 32 ? 256 / L : 1, threads = L <= 32 ? 256 : L;
  const int grid = static_cast<int>((items + per - 1) / per);
  const int ch = (a.part_n / VEC + L - 1) / L;
  if (ch <= 1) gated_norm_kernel<T, VEC, 1, L><<<grid, threads, 0, s>>>(a);
  else if (ch <= 2) gated_norm_kernel<T, VEC, 2, L><<<grid, threads, 0, s>>>(a);
  else gated_norm_kernel<T, VEC, 4, L><<<grid, threads, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int VEC>
int gn_pick(const RbGatedNormArgs& a, cudaStream_t s) {
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.z) | reinterpret_cast<uintptr_t>(a.out);
  const bool vec = !(bits & 15) && !((a.ld_y | a.ld_z | a.ld_o | a.part_n) % VEC);
  if (vec && a.part_n <= 8 * VEC) return gn_launch<T, VEC, 8>(a, s);
  if (vec && a.part_n <= 16 * VEC) return gn_launch<T, VEC, 16>(a, s);
  if (vec && a.part_n <= 32 * VEC * 2) return gn_launch<T, VEC, 32>(a, s);
  if (vec && a.part_n <= 128 * VEC * 2) return gn_launch<T, VEC, 128>(a, s);
  if (vec && a.part_n <= 256 * VEC * 4) return gn_launch<T, VEC, 256>(a, s);
  gated_norm_any_kernel<T><<<a.rows * a.parts, 256, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace rb

RB_API int rb_gated_norm(const RbGatedNormArgs* args, void* stream_v) {
  const RbGatedNormArgs& a = *args;
  if (a.rows <= 0) return 0;
  if (!a.y || !a.z || !a.out || a.parts <= 0 || a.part_n <= 0 ||
      (a.weight_n != a.part_n && a.weight_n != a.parts * a.part_n))
    return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  return a.f32 ? rb::gn_pick<float, 4>(a, s) : rb::gn_pick<__nv_bfloat16, 8>(a, s);
}
