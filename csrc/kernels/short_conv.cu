// Causal convolution over time, one short filter per channel, with silu: the input stage of the recurrent mixers.  One thread
// owns a vector of channels of a tile of 16 rows and slides over them with the last taps - 1 inputs in registers; the tile
// that starts a segment takes those before it from the sequence's state slot and leaves the segment's last inputs there, so
// prompt portions and decoded tokens are one launch.
#include "recurrent.h"

#include "recurrent.cuh"

namespace rb {

constexpr int kScMaxTaps = 16;

template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128)
short_conv_kernel(const RbShortConvArgs a) {
  constexpr int MT = TAPS > 0 ? TAPS : kScMaxTaps;
  const int taps = TAPS > 0 ? TAPS : a.taps;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c >= a.channels) return;
  const int seg = a.tiles[2 * blockIdx.y], off = a.tiles[2 * blockIdx.y + 1];
  const RcSegment s = rc_segment(a.segments, seg, a.num_slots);
  if (off >= s.len) return;
  const int n = min(RB_CONV_TILE, s.len - off);
  const T* x = reinterpret_cast<const T*>(a.x) + static_cast<long long>(s.first + off) * a.ld_x + c;
  T* out = reinterpret_cast<T*>(a.out) + static_cast<long long>(s.first + off) * a.ld_o + c;
  T* st = reinterpret_cast<T*>(a.state) + static_cast<long long>(s.slot) * (taps - 1) * a.channels + c;
  float w[MT][VEC], h[MT][VEC], b[VEC];              // h[i]: the input i + 1 rows before the current one's oldest tap
#pragma unroll
  for (int i = 0; i < MT; ++i) {
#pragma unroll
    for (int v = 0; v < VEC; ++v) { w[i][v] = i < taps ? a.w[static_cast<long long>(c + v) * taps + i] : 0.f; h[i][v] = 0.f; }
  }
#pragma unroll
  for (int v = 0; v < VEC; ++v) b[v] = a.bias ? a.bias[c + v] : 0.f;
  // h[i], i < taps - 1: input at row off - (taps - 1) + i
#pragma unroll
  for (int i = 0; i < MT - 1; ++i) {
    if (i >= taps - 1) break;
    const int back = taps - 1 - i;
    if (off >= back) RcVec<T, VEC>::load(x - back * a.ld_x, h[i]);
    else if (s.start > 0) RcVec<T, VEC>::load(st + static_cast<long long>(taps - 1 - (back - off)) * a.channels, h[i]);
  }
  if (off == 0) {
    // the state behind the segment: its last inputs, or older ones moved up when the segment is shorter than the filter
#pragma unroll
    for (int i = 0; i < MT - 1; ++i) {
      if (i >= taps - 1) break;
      const int r = s.len - (taps - 1) + i;          // row of the segment that becomes entry i
      float u[VEC];
      if (r >= 0) {
        RcVec<T, VEC>::load(x + static_cast<long long>(r) * a.ld_x, u);
      } else {
#pragma unroll
        for (int v = 0; v < VEC; ++v) u[v] = 0.f;
#pragma unroll
        for (int j = 0; j < MT - 1; ++j)             // entry of the old state: r + taps - 1, held in h
          if (j == r + taps - 1) {
#pragma unroll
            for (int v = 0; v < VEC; ++v) u[v] = h[j][v];
          }
      }
      RcVec<T, VEC>::store(st + static_cast<long long>(i) * a.channels, u);
    }
  }
  for (int r = 0; r < n; ++r) {
    float u[VEC], o[VEC];
    RcVec<T, VEC>::load(x + r * a.ld_x, u);
#pragma unroll
    for (int v = 0; v < VEC; ++v) o[v] = b[v];
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      if (i >= taps - 1) break;
#pragma unroll
      for (int v = 0; v < VEC; ++v) o[v] = fmaf(w[i][v], h[i][v], o[v]);
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
      if (i == taps - 1) {
#pragma unroll
        for (int v = 0; v < VEC; ++v) o[v] = fmaf(w[i][v], u[v], o[v]);
      }
#pragma unroll
    for (int i = 0; i < MT - 1; ++i) {
      if (i >= taps - 1) break;
#pragma unroll
      for (int v = 0; v < VEC; ++v) h[i][v] = i == taps - 2 ? u[v] : h[i + 1][v];
    }
    if (a.silu) {
#pragma unroll
      for (int v = 0; v < VEC; ++v) o[v] = rc_silu<T>(o[v]);
    }
    RcVec<T, VEC>::store(out + r * a.ld_o, o);
  }
}

template <typename T, int VEC>
int sc_launch(const RbShortConvArgs& a, cudaStream_t s) {
  const int threads = a.channels / VEC >= 128 ? 128 : 64;
  const dim3 grid((a.channels / VEC + threads - 1) / threads, a.num_tiles);
  switch (a.taps) {
    case 2: short_conv_kernel<T, VEC, 2><<<grid, threads, 0, s>>>(a); break;
    case 3: short_conv_kernel<T, VEC, 3><<<grid, threads, 0, s>>>(a); break;
    case 4: short_conv_kernel<T, VEC, 4><<<grid, threads, 0, s>>>(a); break;
    default: short_conv_kernel<T, 1, 0><<<dim3((a.channels + threads - 1) / threads, a.num_tiles), threads, 0, s>>>(a);
  }
  return static_cast<int>(cudaGetLastError());
}

}  // namespace rb

RB_API int rb_short_conv(const RbShortConvArgs* args, void* stream_v) {
  const RbShortConvArgs& a = *args;
  if (a.num_tiles <= 0) return 0;
  if (!a.x || !a.out || !a.w || !a.segments || !a.tiles || a.channels <= 0 || a.taps < 1 || a.taps > rb::kScMaxTaps ||
      a.num_slots <= 0 || (a.taps > 1 && !a.state) || a.num_tiles > 65535)
    return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_v);
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.out) | reinterpret_cast<uintptr_t>(a.state);
  const long long n = a.channels | a.ld_x | a.ld_o;
  if (a.f32) return !(bits & 15) && !(n & 3) ? rb::sc_launch<float, 4>(a, s) : rb::sc_launch<float, 1>(a, s);
  return !(bits & 7) && !(n & 3) ? rb::sc_launch<__nv_bfloat16, 4>(a, s) : rb::sc_launch<__nv_bfloat16, 1>(a, s);
}
