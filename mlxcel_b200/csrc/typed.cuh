// Element access shared by the kernels that exist for bf16 and for fp32 activations: scalar and
// four-element loads / stores that widen to and narrow from fp32.
#pragma once
#include "common.cuh"

namespace mx {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// V consecutive elements (V = 1 or 4; the four-element form needs an address aligned to the group).
template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    f[0] = a.x, f[1] = a.y, f[2] = a.z, f[3] = a.w;
  } else {
    f[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void load_v(const __nv_bfloat16* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    f[0] = bf16_lo(a.x), f[1] = bf16_hi(a.x), f[2] = bf16_lo(a.y), f[3] = bf16_hi(a.y);
  } else {
    f[0] = __bfloat162float(*p);
  }
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float (&f)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else *p = f[0];
}
template <int V>
__device__ __forceinline__ void store_v(__nv_bfloat16* p, const float (&f)[V]) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]));
  else *p = __float2bfloat16(f[0]);
}

inline bool aligned_to(const void* p, size_t bytes) { return reinterpret_cast<uintptr_t>(p) % bytes == 0; }

// Sum of N values over the CTA (every thread receives the totals). `red` holds 33 * N floats.
template <int N>
__device__ __forceinline__ void block_sums(float (&v)[N], float* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = (blockDim.x + 31) >> 5;
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_sum(v[i]);
  __syncthreads();                       // a previous round's totals have been read
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) red[i * 33 + warp] = v[i];
  }
  __syncthreads();
  if (warp == 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const float t = warp_sum(lane < warps ? red[i * 33 + lane] : 0.f);
      if (lane == 0) red[i * 33 + 32] = t;
    }
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = red[i * 33 + 32];
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

}  // namespace mx
