// moe_route.cuh -- the choice of a sigmoid router with a correction and group-limited top-k for ONE row, by one warp, and the rider of
// a norm in front of a mixture of experts (RouteRider, nogatar.h) that works out the row's logits first.
#pragma once
#include "common.cuh"
#include "nogatar.h"

namespace qie {

// the largest value, the lowest index among equals; every lane returns the winner
__device__ __forceinline__ int warp_argmax_first(const float* v, int count, int lane) {
  float bv = -INFINITY;
  int bi = 0x7fffffff;
  for (int e = lane; e < count; e += 32) {
    const float x = v[e];
    if (bi == 0x7fffffff || x > bv) bv = x, bi = e;  // ascending e within a lane
  }
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (oi != 0x7fffffff && (bi == 0x7fffffff || ov > bv || (ov == bv && oi < bi))) bv = ov, bi = oi;
  }
  return bi;
}

// floats of scratch the warp needs: choice scores [experts] | plain scores [experts] | group scores [groups] | kept marks [groups]
__host__ __device__ inline size_t route_scratch_floats(int experts, int groups) { return (size_t)2 * experts + 2 * (size_t)groups; }

// z: the row's router logits (any memory the warp can read); scratch: route_scratch_floats() floats of shared memory
__device__ __forceinline__ void route_sigmoid_row(const float* z, float* scratch, int experts, int top, int groups, int keep,
                                                  const bf16* __restrict__ correction, float scale, int* __restrict__ top_idx,
                                                  float* __restrict__ top_w, int lane) {
  float* c = scratch;
  float* s = c + experts;
  float* gs = s + experts;
  float* kept = gs + groups;
  for (int e = lane; e < experts; e += 32) {
    const float v = 1.0f / (1.0f + expf(-z[e]));
    s[e] = v;
    // the choice scores; where nothing is added to a score its logit orders the experts alike, also where the sigmoid saturates
    c[e] = correction ? v + bf2f(correction[e]) : keep < groups ? v : z[e];
  }
  __syncwarp();
  if (keep < groups) {
    const int per = experts / groups;
    for (int g = lane; g < groups; g += 32) {  // the two largest choice scores of the group
      float a = -INFINITY, b = -INFINITY;
      for (int e = g * per; e < (g + 1) * per; ++e) {
        const float x = c[e];
        if (x > a) b = a, a = x;
        else if (x > b) b = x;
      }
      gs[g] = per > 1 ? a + b : a;
      kept[g] = 0.f;
    }
    __syncwarp();
    for (int k = 0; k < keep; ++k) {
      const int bi = warp_argmax_first(gs, groups, lane);
      __syncwarp();
      if (lane == 0) gs[bi] = -INFINITY, kept[bi] = 1.f;
      __syncwarp();
    }
    // experts of the other groups drop out of the choice (not merely to zero: choice scores may be negative)
    for (int e = lane; e < experts; e += 32)
      if (kept[e / per] == 0.f) c[e] = -INFINITY;
    __syncwarp();
  }
  for (int k = 0; k < top; ++k) {
    const int bi = warp_argmax_first(c, experts, lane);
    __syncwarp();
    if (lane == 0) {
      top_idx[k] = bi;
      top_w[k] = s[bi] * scale;
      c[bi] = -INFINITY;
    }
    __syncwarp();
  }
}

// the rider of a norm kernel (RouteRider): the CTA of row r holds the normed row h [W] in shared memory (complete) and works out the
// router's logits, a warp per two experts, lanes striding the width (four elements at a time when the rows allow it); warp 0 then chooses.  h is
// 16-byte aligned.
// zl: experts + route_scratch_floats() floats of shared memory
__device__ __forceinline__ void route_rider_row(const RouteRider& rt, int r, const float* h, int W, float* zl) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const bool vec = W % 4 == 0 && (reinterpret_cast<uintptr_t>(rt.w_router) & 7) == 0;
  for (int e = warp; e < rt.experts; e += 2 * nw) {  // two experts at a time share the reads of the row
    const int e2 = e + nw;
    const bool two = e2 < rt.experts;
    const bf16 *wa = rt.w_router + (size_t)e * W, *wb = rt.w_router + (size_t)(two ? e2 : e) * W;
    float acc = 0.f, acc2 = 0.f;
    if (vec) {
#pragma unroll 8
      for (int i = lane * 4; i < W; i += 128) {
        const uint2 p = *reinterpret_cast<const uint2*>(wa + i), q = *reinterpret_cast<const uint2*>(wb + i);
        const float4 x = *reinterpret_cast<const float4*>(h + i);
        acc = fmaf(x.x, lo2f(p.x), acc), acc = fmaf(x.y, hi2f(p.x), acc), acc = fmaf(x.z, lo2f(p.y), acc), acc = fmaf(x.w, hi2f(p.y), acc);
        acc2 = fmaf(x.x, lo2f(q.x), acc2), acc2 = fmaf(x.y, hi2f(q.x), acc2), acc2 = fmaf(x.z, lo2f(q.y), acc2), acc2 = fmaf(x.w, hi2f(q.y), acc2);
      }
    } else {
      for (int i = lane; i < W; i += 32) acc = fmaf(h[i], bf2f(wa[i]), acc), acc2 = fmaf(h[i], bf2f(wb[i]), acc2);
    }
    acc = warp_sum(acc), acc2 = warp_sum(acc2);
    if (lane == 0) {
      zl[e] = acc;
      if (two) zl[e2] = acc2;
    }
  }
  __syncthreads();
  if (warp == 0)
    route_sigmoid_row(zl, zl + rt.experts, rt.experts, rt.top, rt.groups, rt.keep, rt.correction, rt.scale, rt.top_idx + (size_t)r * rt.top,
                      rt.top_w + (size_t)r * rt.top, lane);
}

}  // namespace qie
