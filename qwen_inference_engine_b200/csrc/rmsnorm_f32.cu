// rmsnorm_f32.cu -- RMS norms of a model whose sublayers sit between two norms (ditenex.h): the output norm folded
// into the residual add together with the next sublayer's input norm, and the input norm of a mixer that reads a blend
// of each row with the row before it (token shift) with one carried row per sequence slot; and the grouped RMS norm of a
// model of parallel blocks (dedunex.h): the residual add of the two sublayer outputs and the next block's norm in one kernel;
// and the grouped norm with a gate behind it (gebadra.h).  A model with one group and a router in front of its experts (gubanex.h) uses
// the grouped step with the router's rider.
// All fp32, one CTA per row, every reduction in a fixed order per row, so a row's result does not depend on the rows it
// shares a launch with.
#include "dedunex.h"
#include "ditenex.h"
#include "gebadra.h"
#include "launch.h"
#include "moe_route.cuh"
#include "pack.cuh"

namespace qie {
namespace {

template <int V>
__global__ void __launch_bounds__(256) rms_step_kernel(const RmsStep a) {
  extern __shared__ __align__(16) float row[];  // [width]
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, W = a.width;
  const int t0 = threadIdx.x * V, step = blockDim.x * V;
  const bool add = a.y || a.y_bf || a.mix.ye;
  const int src = a.gather ? a.gather[r] : r;  // the add half is never combined with a gather
  float* xr = a.x + (size_t)src * W;
  float sq = 0.f;
  if (add) {
    float s = 0.f;
    if (a.y || a.y_bf) {
      for (int i = t0; i < W; i += step) {
        const Pack<V> p = a.y_bf ? ld_bf16<V>(a.y_bf + (size_t)r * W + i) : ld_f32<V>(a.y + (size_t)r * W + i);
        st_f32<V>(row + i, p);
#pragma unroll
        for (int u = 0; u < V; ++u) s = fmaf(p.v[u], p.v[u], s);
      }
    } else {  // the chosen experts' outputs of this row, weighted, plus the shared expert (gated only when mix.z is given)
      const MoeMix& m = a.mix;
      const bool shared = m.ys || a.ys_bf;
      const float sg = shared ? (m.z ? 1.0f / (1.0f + expf(-m.z[(size_t)r * m.ldz + m.gate_col])) : 1.0f) : 0.f;
      for (int i = t0; i < W; i += step) {
        Pack<V> p;
#pragma unroll
        for (int u = 0; u < V; ++u) p.v[u] = 0.f;
        for (int k = 0; k < m.top; ++k) {
          const float wk = m.top_w[(size_t)r * m.top + k];
          const Pack<V> e = ld_f32<V>(m.ye + (size_t)m.slot_of[(size_t)r * m.top + k] * W + i);
#pragma unroll
          for (int u = 0; u < V; ++u) p.v[u] = fmaf(wk, e.v[u], p.v[u]);
        }
        if (shared) {
          const Pack<V> e = a.ys_bf ? ld_bf16<V>(a.ys_bf + (size_t)r * W + i) : ld_f32<V>(m.ys + (size_t)r * W + i);
#pragma unroll
          for (int u = 0; u < V; ++u) p.v[u] = fmaf(sg, e.v[u], p.v[u]);
        }
        st_f32<V>(row + i, p);
#pragma unroll
        for (int u = 0; u < V; ++u) s = fmaf(p.v[u], p.v[u], s);
      }
    }
    const float rstd = 1.0f / sqrtf(block_sum_r(s, red) / (float)W + a.eps);
    for (int i = t0; i < W; i += step) {
      const Pack<V> y = ld_f32<V>(row + i), x = ld_f32<V>(xr + i), w = ld_bf16<V>(a.w_out + i);
      Pack<V> o;
#pragma unroll
      for (int u = 0; u < V; ++u) {
        o.v[u] = x.v[u] + a.mult * (y.v[u] * rstd * w.v[u]);
        sq = fmaf(o.v[u], o.v[u], sq);
      }
      st_f32<V>(xr + i, o);
      st_f32<V>(row + i, o);
    }
  } else if (a.h || a.h_bf) {
    for (int i = t0; i < W; i += step) {
      const Pack<V> x = ld_f32<V>(xr + i);
      st_f32<V>(row + i, x);
#pragma unroll
      for (int u = 0; u < V; ++u) sq = fmaf(x.v[u], x.v[u], sq);
    }
  }
  if (!a.h && !a.h_bf) return;
  const float rstd = 1.0f / sqrtf(block_sum_r(sq, red) / (float)W + a.eps);
  for (int i = t0; i < W; i += step) {
    const Pack<V> x = ld_f32<V>(row + i), w = ld_bf16<V>(a.w_in + i);
    Pack<V> o;
#pragma unroll
    for (int u = 0; u < V; ++u) o.v[u] = x.v[u] * rstd * w.v[u];
    if (a.h) st_f32<V>(a.h + (size_t)r * W + i, o);
    if (a.h_bf) st_bf16<V>(a.h_bf + (size_t)r * W + i, o);
    st_f32<V>(row + i, o);
  }
  if (!a.route.w_router) return;
  __syncthreads();  // the normed row is complete
  route_rider_row(a.route, r, row, W, row + W);
}

// one CTA per row.  The CTA of a segment's first row also moves the segment's last normed row into the carried row:
// each thread reads the old carried elements it needs before it overwrites exactly those, and no other CTA touches them.
template <int V>
__global__ void __launch_bounds__(256) rms_shift_kernel(const RmsShiftArgs a) {
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, W = a.width;
  const int t0 = threadIdx.x * V, step = blockDim.x * V;
  // the segment of this row: the last s with seg_start[s] <= r
  int lo = 0, hi = a.n_seg - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (a.seg_start[mid] <= r) lo = mid;
    else hi = mid - 1;
  }
  const int first = a.seg_start[lo], last = a.seg_start[lo + 1] - 1;
  const bool head = r == first;
  const float* xr = a.x + (size_t)r * W;
  const float* xp = head ? a.x + (size_t)last * W : xr - W;  // the other row this CTA norms: the one before, or (first row) the segment's last
  float s0 = 0.f, s1 = 0.f;
  for (int i = t0; i < W; i += step) {
    const Pack<V> v = ld_f32<V>(xr + i), u = ld_f32<V>(xp + i);
#pragma unroll
    for (int k = 0; k < V; ++k) s0 = fmaf(v.v[k], v.v[k], s0), s1 = fmaf(u.v[k], u.v[k], s1);
  }
  const float r0 = 1.0f / sqrtf(block_sum_r(s0, red) / (float)W + a.eps);
  const float r1 = 1.0f / sqrtf(block_sum_r(s1, red) / (float)W + a.eps);
  float* carry = a.carry + (size_t)a.seg_slot[lo] * a.slot_stride;
  for (int i = t0; i < W; i += step) {
    const Pack<V> v = ld_f32<V>(xr + i), u = ld_f32<V>(xp + i), w = ld_bf16<V>(a.w + i), mu = ld_bf16<V>(a.mu + i);
    Pack<V> before, o, res;
    if (head) before = ld_f32<V>(carry + i);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const float h = v.v[k] * r0 * w.v[k];
      o.v[k] = u.v[k] * r1 * w.v[k];
      const float b = head ? before.v[k] : o.v[k];
      res.v[k] = h + (b - h) * mu.v[k];
    }
    if (a.out) st_f32<V>(a.out + (size_t)r * W + i, res);
    if (a.out_bf) st_bf16<V>(a.out_bf + (size_t)r * W + i, res);
    if (head) st_f32<V>(carry + i, o);
  }
}


// The row lies in shared memory.  Each of the `groups` parts is normed by a team of warps: with fewer groups than warps a
// group gets blockDim / 32 / groups warps whose partial sums meet in shared memory in a fixed order, else a warp walks the
// groups warp, warp + nw, ...  scale[g] receives 1 / sqrt(mean + eps) of every group.
__device__ __forceinline__ void group_rstd(const float* row, int W, int groups, float eps, float* red, float* scale) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5, gs = W / groups;
  if (groups >= nw) {
    for (int g = warp; g < groups; g += nw) {
      float s = 0.f;
      for (int i = lane; i < gs; i += 32) s = fmaf(row[g * gs + i], row[g * gs + i], s);
      s = warp_sum(s);
      if (lane == 0) scale[g] = 1.0f / sqrtf(s / (float)gs + eps);
    }
  } else {
    const int wpg = nw / groups, g = warp / wpg, k = warp % wpg;
    float s = 0.f;
    if (g < groups)
      for (int i = k * 32 + lane; i < gs; i += 32 * wpg) s = fmaf(row[g * gs + i], row[g * gs + i], s);
    s = warp_sum(s);
    if (lane == 0) red[warp] = s;
    __syncthreads();
    if (threadIdx.x < groups) {
      float t = 0.f;
      for (int j = 0; j < wpg; ++j) t += red[threadIdx.x * wpg + j];
      scale[threadIdx.x] = 1.0f / sqrtf(t / (float)gs + eps);
    }
  }
  __syncthreads();
}

// NR > 0: one group, the row stays in NR packs of registers per thread; NR = 0: any number of groups, the row in shared memory
template <int V, int NR>
__global__ void __launch_bounds__(256) group_norm_step_kernel(const GroupNormStep a) {
  extern __shared__ __align__(16) float row[];  // [width], then [groups] scales, then the router's logits and scratch
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, W = a.width, gs = W / a.groups;
  float* scale = row + W;
  const int t0 = threadIdx.x * V, step = blockDim.x * V;
  const int src = a.gather ? a.gather[r] : r;
  float* xr = a.x + (size_t)src * W;
  const bf16* entry = a.ids ? a.embed + (size_t)a.ids[src] * W : nullptr;
  const bool fresh = a.ids && !a.again, normed = fresh && a.w_pre;
  const bool has1 = a.y1 || a.y1_bf, has2 = a.y2 || a.y2_bf, mixed = a.mix.ye || a.ye_bf;
  const bool changed = a.ids || has1 || has2 || mixed || a.step;
  if (normed) {  // the embedding row, normed
    for (int i = t0; i < W; i += step) st_f32<V>(row + i, ld_bf16<V>(entry + i));
    __syncthreads();
    group_rstd(row, W, a.groups, a.eps, red, scale);
  }
  auto entry_at = [&](int i) {
    Pack<V> v = ld_bf16<V>(entry + i);
#pragma unroll
    for (int u = 0; u < V; ++u) v.v[u] *= a.embed_scale;
    return v;
  };
  // elements i .. i + V - 1 of the stream after every addition; a thread touches only its own elements of the row
  auto value = [&](int i) {
    Pack<V> v;
    if (normed) {
      v = ld_f32<V>(row + i);
      const Pack<V> w = ld_bf16<V>(a.w_pre + i);
#pragma unroll
      for (int u = 0; u < V; ++u) v.v[u] = v.v[u] * scale[(i + u) / gs] * w.v[u];
    } else {
      v = fresh ? entry_at(i) : ld_f32<V>(xr + i);
    }
    if (has1 || has2) {
      Pack<V> y, z;
      if (has1) y = a.y1_bf ? ld_bf16<V>(a.y1_bf + (size_t)src * W + i) : ld_f32<V>(a.y1 + (size_t)src * W + i);
      if (has2) z = a.y2_bf ? ld_bf16<V>(a.y2_bf + (size_t)src * W + i) : ld_f32<V>(a.y2 + (size_t)src * W + i);
#pragma unroll
      for (int u = 0; u < V; ++u) v.v[u] += has1 && has2 ? y.v[u] + z.v[u] : has1 ? y.v[u] : z.v[u];
    }
    if (mixed) {
      Pack<V> s;
#pragma unroll
      for (int u = 0; u < V; ++u) s.v[u] = 0.f;
      for (int k = 0; k < a.mix.top; ++k) {
        const size_t at = (size_t)src * a.mix.top + k, o = (size_t)a.mix.slot_of[at] * W + i;
        const float wk = a.mix.top_w ? a.mix.top_w[at] : 1.0f;
        const Pack<V> e = a.ye_bf ? ld_bf16<V>(a.ye_bf + o) : ld_f32<V>(a.mix.ye + o);
#pragma unroll
        for (int u = 0; u < V; ++u) s.v[u] = fmaf(wk, e.v[u], s.v[u]);
      }
#pragma unroll
      for (int u = 0; u < V; ++u) v.v[u] += s.v[u];
    }
    if (a.dump) st_f32<V>(a.dump + (size_t)r * W + i, v);
    if (a.step) {
      const Pack<V> s = ld_bf16<V>(a.step + i);
#pragma unroll
      for (int u = 0; u < V; ++u) v.v[u] += s.v[u];
    }
    if (a.again) {
      const Pack<V> s = entry_at(i);
#pragma unroll
      for (int u = 0; u < V; ++u) v.v[u] += s.v[u];
    }
    if (changed) st_f32<V>(xr + i, v);
    return v;
  };
  const bool read = a.h || a.h_bf;
  auto emit = [&](int i, const Pack<V>& x, const Pack<V>& w, float s0) {
    Pack<V> o;
#pragma unroll
    for (int u = 0; u < V; ++u) o.v[u] = x.v[u] * (NR > 0 ? s0 : scale[(i + u) / gs]) * (a.w_off + w.v[u]);
    if (a.h) st_f32<V>(a.h + (size_t)r * W + i, o);
    if (a.h_bf) st_bf16<V>(a.h_bf + (size_t)r * W + i, o);
    if (a.route.w_router) st_f32<V>(row + i, o);
  };
  if (!read) {
    for (int i = t0; i < W; i += step) value(i);
    return;
  }
  if constexpr (NR > 0) {
    Pack<V> x[NR], w[NR];
    float sq = 0.f;
#pragma unroll
    for (int k = 0; k < NR; ++k)
      if (t0 + k * step < W) x[k] = value(t0 + k * step), w[k] = ld_bf16<V>(a.w_in + t0 + k * step);
#pragma unroll
    for (int k = 0; k < NR; ++k)
      if (t0 + k * step < W)
#pragma unroll
        for (int u = 0; u < V; ++u) sq = fmaf(x[k].v[u], x[k].v[u], sq);
    const float s0 = 1.0f / sqrtf(block_sum_r(sq, red) / (float)W + a.eps);
#pragma unroll
    for (int k = 0; k < NR; ++k)
      if (t0 + k * step < W) emit(t0 + k * step, x[k], w[k], s0);
  } else {
    for (int i = t0; i < W; i += step) st_f32<V>(row + i, value(i));
    __syncthreads();
    group_rstd(row, W, a.groups, a.eps, red, scale);
    for (int i = t0; i < W; i += step) emit(i, ld_f32<V>(row + i), ld_bf16<V>(a.w_in + i), 0.f);
  }
  if (!a.route.w_router) return;
  __syncthreads();  // the normed row is complete
  route_rider_row(a.route, r, row, W, scale + a.groups);
}

template <int V>
__global__ void __launch_bounds__(256) norm_gate_kernel(const NormGate a) {
  extern __shared__ __align__(16) float row[];  // [width], then [groups] scales
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const size_t r = blockIdx.x;
  const int W = a.width, gs = W / a.groups, t0 = threadIdx.x * V, step = blockDim.x * V;
  float* scale = row + W;
  auto gate_of = [&](int i) { return a.g_bf ? ld_bf16<V>(a.g_bf + r * a.ldg_bf + i) : ld_f32<V>(a.g + r * a.ldg + i); };
  auto finish = [&](int i, Pack<V> x, const Pack<V>& g, float s0) {
    Pack<V> w;
    if (a.w) w = ld_bf16<V>(a.w + (a.w_shared ? i % gs : i));
#pragma unroll
    for (int u = 0; u < V; ++u) {
      const float sg = 1.0f / (1.0f + expf(-g.v[u]));
      float y = x.v[u] * (a.groups == 1 ? s0 : scale[(i + u) / gs]);
      if (a.w) y *= w.v[u];
      x.v[u] = y * (a.act == 1 ? sg : g.v[u] * sg);
    }
    if (a.out) st_f32<V>(a.out + r * a.ldo + i, x);
    if (a.out_bf) st_bf16<V>(a.out_bf + r * a.ldo_bf + i, x);
  };
  constexpr int NR = 2;
  if (a.groups == 1 && W <= NR * step) {  // the row and its gate stay in registers, every load in flight at once
    Pack<V> x[NR], g[NR];
    float sq = 0.f;
#pragma unroll
    for (int k = 0; k < NR; ++k)
      if (t0 + k * step < W) x[k] = ld_f32<V>(a.v + r * a.ldv + t0 + k * step), g[k] = gate_of(t0 + k * step);
#pragma unroll
    for (int k = 0; k < NR; ++k)
      if (t0 + k * step < W)
#pragma unroll
        for (int u = 0; u < V; ++u) sq = fmaf(x[k].v[u], x[k].v[u], sq);
    const float s0 = 1.0f / sqrtf(block_sum_r(sq, red) / (float)W + a.eps);
#pragma unroll
    for (int k = 0; k < NR; ++k)
      if (t0 + k * step < W) finish(t0 + k * step, x[k], g[k], s0);
    return;
  }
  for (int i = t0; i < W; i += step) st_f32<V>(row + i, ld_f32<V>(a.v + r * a.ldv + i));
  __syncthreads();
  group_rstd(row, W, a.groups, a.eps, red, scale);
  for (int i = t0; i < W; i += step) finish(i, ld_f32<V>(row + i), gate_of(i), scale[0]);
}

}  // namespace

cudaError_t launch_norm_gate(const NormGate& a, cudaStream_t st) {
  if (a.n <= 0) return cudaSuccess;
  if (a.width <= 0 || a.groups <= 0 || a.width % a.groups || !a.v || !(a.g || a.g_bf) || !(a.out || a.out_bf)) return cudaErrorInvalidValue;
  const size_t smem = ((size_t)a.width + a.groups) * sizeof(float);
  auto al = [](const void* p, size_t b) { return (reinterpret_cast<uintptr_t>(p) & (b - 1)) == 0; };
  const bool vec = a.width % 4 == 0 && (!a.w_shared || a.width / a.groups % 4 == 0) && a.ldv % 4 == 0 && a.ldg % 4 == 0 && a.ldg_bf % 4 == 0 && a.ldo % 4 == 0 && a.ldo_bf % 4 == 0 && al(a.v, 16) &&
                   al(a.g, 16) && al(a.g_bf, 8) && al(a.w, 8) && al(a.out, 16) && al(a.out_bf, 8);
  auto* kern = vec ? norm_gate_kernel<4> : norm_gate_kernel<1>;
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) return cudaErrorInvalidValue;
    cudaError_t r = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (r != cudaSuccess) return r;
  }
  return launch_k(kern, dim3(a.n), dim3(256), smem, st, a);
}

static bool route_ok(const RouteRider& rt) {
  return rt.experts > 0 && rt.top > 0 && rt.top <= rt.experts && rt.groups > 0 && rt.experts % rt.groups == 0 && rt.keep > 0 && rt.keep <= rt.groups && rt.top_idx &&
         rt.top_w;
}

cudaError_t launch_group_norm_step(const GroupNormStep& a, cudaStream_t st) {
  if (a.n <= 0) return cudaSuccess;
  const bool read = a.h || a.h_bf;
  if (a.width <= 0 || a.groups <= 0 || a.width % a.groups || (read && !a.w_in) || (a.ids && (!a.embed || a.gather)) || (a.again && (!a.ids || a.w_pre))) return cudaErrorInvalidValue;
  size_t smem = ((size_t)a.width + a.groups) * sizeof(float);
  if (a.route.w_router) {
    if (!read || a.gather || !route_ok(a.route)) return cudaErrorInvalidValue;
    smem += ((size_t)a.route.experts + route_scratch_floats(a.route.experts, a.route.groups)) * sizeof(float);
  }
  auto al = [](const void* p, size_t b) { return (reinterpret_cast<uintptr_t>(p) & (b - 1)) == 0; };
  const bool vec = a.width % 4 == 0 && al(a.x, 16) && al(a.y1, 16) && al(a.y2, 16) && al(a.y1_bf, 8) && al(a.y2_bf, 8) && al(a.mix.ye, 16) && al(a.ye_bf, 8) &&
                   al(a.dump, 16) && al(a.h, 16) && al(a.h_bf, 8) && al(a.w_in, 8) && al(a.w_pre, 8) && al(a.step, 8) && al(a.embed, 8);
  const bool regs = vec && a.groups == 1 && !(a.ids && a.w_pre);
  auto* kern = !vec ? group_norm_step_kernel<1, 0> : !regs ? group_norm_step_kernel<4, 0> : a.width <= 1024 ? group_norm_step_kernel<4, 1>
               : a.width <= 2048 ? group_norm_step_kernel<4, 2> : a.width <= 4096 ? group_norm_step_kernel<4, 4> : group_norm_step_kernel<4, 0>;
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) return cudaErrorInvalidValue;
    cudaError_t r = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (r != cudaSuccess) return r;
  }
  return launch_k(kern, dim3(a.n), dim3(256), smem, st, a);
}

cudaError_t launch_rms_step(const RmsStep& a, cudaStream_t st) {
  if (a.n <= 0) return cudaSuccess;
  const bool add = a.y || a.y_bf || a.mix.ye, read = a.h || a.h_bf;
  if ((add && (!a.w_out || a.gather)) || (read && !a.w_in) || (!add && !read)) return cudaErrorInvalidValue;
  size_t smem = (size_t)a.width * sizeof(float);
  if (a.route.w_router) {
    const RouteRider& rt = a.route;
    if (!read || a.gather || !route_ok(rt)) return cudaErrorInvalidValue;
    smem += ((size_t)rt.experts + route_scratch_floats(rt.experts, rt.groups)) * sizeof(float);
  }
  // 16-byte accesses when every row starts on a 16-byte boundary (cudaMalloc'd buffers, width a multiple of 4)
  auto al = [](const void* p, size_t b) { return (reinterpret_cast<uintptr_t>(p) & (b - 1)) == 0; };
  const bool vec = a.width % 4 == 0 && al(a.x, 16) && al(a.y, 16) && al(a.y_bf, 8) && al(a.ys_bf, 8) && al(a.mix.ye, 16) && al(a.mix.ys, 16) &&
                   al(a.h, 16) && al(a.h_bf, 8) && al(a.w_out, 8) && al(a.w_in, 8);
  auto* kern = vec ? rms_step_kernel<4> : rms_step_kernel<1>;
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) return cudaErrorInvalidValue;
    cudaError_t r = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (r != cudaSuccess) return r;
  }
  return launch_k(kern, dim3(a.n), dim3(256), smem, st, a);
}

cudaError_t launch_rms_shift(const RmsShiftArgs& a, cudaStream_t st) {
  if (a.n <= 0) return cudaSuccess;
  if (a.n_seg <= 0 || !a.seg_start || !a.seg_slot || !a.carry) return cudaErrorInvalidValue;
  auto al = [](const void* p, size_t b) { return (reinterpret_cast<uintptr_t>(p) & (b - 1)) == 0; };
  const bool vec = a.width % 4 == 0 && a.slot_stride % 4 == 0 && al(a.x, 16) && al(a.out, 16) && al(a.out_bf, 8) && al(a.carry, 16) && al(a.w, 8) &&
                   al(a.mu, 8);
  return vec ? launch_k(rms_shift_kernel<4>, dim3(a.n), dim3(256), 0, st, a) : launch_k(rms_shift_kernel<1>, dim3(a.n), dim3(256), 0, st, a);
}

}  // namespace qie
