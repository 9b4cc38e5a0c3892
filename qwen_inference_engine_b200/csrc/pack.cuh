// pack.cuh -- V consecutive elements per thread and step of a row kernel (V = 4: 16-byte fp32 and 8-byte bf16 accesses
// when the width and the pointers allow it; V = 1 otherwise), and the fixed-order block sums of such kernels.
#pragma once
#include "common.cuh"

namespace qie {

template <int V>
struct Pack {
  float v[V];
};
template <int V>
__device__ __forceinline__ Pack<V> ld_f32(const float* p) {
  Pack<V> r;
  if constexpr (V == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    r.v[0] = t.x, r.v[1] = t.y, r.v[2] = t.z, r.v[3] = t.w;
  } else {
    r.v[0] = p[0];
  }
  return r;
}
template <int V>
__device__ __forceinline__ Pack<V> ld_bf16(const bf16* p) {
  Pack<V> r;
  if constexpr (V == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    r.v[0] = lo2f(t.x), r.v[1] = hi2f(t.x), r.v[2] = lo2f(t.y), r.v[3] = hi2f(t.y);
  } else {
    r.v[0] = bf2f(p[0]);
  }
  return r;
}
template <int V>
__device__ __forceinline__ void st_f32(float* p, const Pack<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else p[0] = r.v[0];
}
template <int V>
__device__ __forceinline__ void st_bf16(bf16* p, const Pack<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack2(f2bf(r.v[0]), f2bf(r.v[1])), pack2(f2bf(r.v[2]), f2bf(r.v[3])));
  else p[0] = f2bf(r.v[0]);
}

// sum over the block, the same in every thread; red holds 32 floats
__device__ __forceinline__ float block_sum_r(float v, float* red) {
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();  // red may still be read from the previous call
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = l < nw ? red[l] : 0.f;
  for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
  return t;
}
// two sums at once; red holds 64 floats
__device__ __forceinline__ float2 block_sum2_r(float a, float b, float* red) {
  for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o), b += __shfl_xor_sync(0xffffffffu, b, o);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (l == 0) red[w] = a, red[32 + w] = b;
  __syncthreads();
  float s = l < nw ? red[l] : 0.f, t = l < nw ? red[32 + l] : 0.f;
  for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o), t += __shfl_xor_sync(0xffffffffu, t, o);
  return make_float2(s, t);
}

}  // namespace qie
