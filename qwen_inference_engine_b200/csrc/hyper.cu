// hyper.cu -- hyper-connections: a model that carries `streams` copies of the residual stream.  A sublayer reads a
// learned combination of the streams (then an RMS norm or a layer norm), and writes back by mixing the streams with a
// learned matrix and adding its output -- or the sum of the RMS-normed outputs of two sublayers side by side -- with a
// learned factor per stream.  One kernel does a sublayer's write and the next sublayer's read + norm, one CTA per row;
// all arithmetic is fp32 and every reduction has a fixed order per row.
#include "fosavik.h"
#include "launch.h"
#include "pack.cuh"

namespace qie {
namespace {

constexpr int HC_MAX_STREAMS = 8;

__global__ void embed_streams_kernel(float* __restrict__ X, const bf16* __restrict__ embed, const bf16* __restrict__ pos_table,
                                     const int* __restrict__ ids, const int* __restrict__ pos, int width, int streams) {
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x;
  const bf16* src = embed + (size_t)ids[r] * width;
  const bf16* pp = pos_table ? pos_table + (size_t)pos[r] * width : nullptr;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float v = bf2f(src[i]) + (pp ? bf2f(pp[i]) : 0.f);
    for (int s = 0; s < streams; ++s) X[((size_t)r * streams + s) * width + i] = v;
  }
}

template <int S, int V>
__global__ void __launch_bounds__(256) hyper_step_kernel(const HyperStep a) {
  extern __shared__ __align__(16) float row[];  // [width] what the read half norms
  __shared__ float red[64];
  __shared__ float mix[S * S], outv[S], inv[S];
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x;
  const int W = a.width;
  const int t0 = threadIdx.x * V, step = blockDim.x * V;
  const bool write = a.y1 || a.y1_bf, two = a.y2 || a.y2_bf;
  if (write && threadIdx.x < S * S) mix[threadIdx.x] = bf2f(a.mix[threadIdx.x]);
  if (threadIdx.x < S) {
    if (write) outv[threadIdx.x] = bf2f(a.out[threadIdx.x]);
    inv[threadIdx.x] = a.in ? bf2f(a.in[threadIdx.x]) : 1.0f;
  }
  __syncthreads();
  auto y1 = [&](int i) { return a.y1_bf ? ld_bf16<V>(a.y1_bf + (size_t)r * W + i) : ld_f32<V>(a.y1 + (size_t)r * W + i); };
  auto y2 = [&](int i) { return a.y2_bf ? ld_bf16<V>(a.y2_bf + (size_t)r * W + i) : ld_f32<V>(a.y2 + (size_t)r * W + i); };
  float f1 = a.s1, f2 = a.s2;
  if (write && a.y1_norm) {  // the outputs are normed over the width before they are added
    float q1 = 0.f, q2 = 0.f;
    for (int i = t0; i < W; i += step) {
      const Pack<V> p = y1(i);
#pragma unroll
      for (int u = 0; u < V; ++u) q1 = fmaf(p.v[u], p.v[u], q1);
      if (two) {
        const Pack<V> q = y2(i);
#pragma unroll
        for (int u = 0; u < V; ++u) q2 = fmaf(q.v[u], q.v[u], q2);
      }
    }
    const float2 s = block_sum2_r(q1, q2, red);
    f1 *= 1.0f / sqrtf(s.x / (float)W + a.eps);
    f2 *= 1.0f / sqrtf(s.y / (float)W + a.eps);
  }
  const int src = a.gather ? a.gather[r] : r;  // the write half is never combined with a gather
  float* Xr = a.X + (size_t)src * S * W;
  const bf16* er = a.ids ? a.embed + (size_t)a.ids[r] * W : nullptr;
  const bool read = a.h || a.h_bf;
  float sum = 0.f;  // of u (layer norm) or of u^2 (RMS norm)
  for (int i = t0; i < W; i += step) {
    Pack<V> x[S];
    if (er) {
      x[0] = ld_bf16<V>(er + i);
#pragma unroll
      for (int s = 0; s < S; ++s) {
        if (s) x[s] = x[0];
        st_f32<V>(Xr + (size_t)s * W + i, x[0]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) x[s] = ld_f32<V>(Xr + (size_t)s * W + i);
    }
    if (write) {
      Pack<V> y = y1(i);
      if (a.y1_norm) {
        const Pack<V> w = ld_bf16<V>(a.y1_norm + i);
#pragma unroll
        for (int u = 0; u < V; ++u) y.v[u] *= w.v[u];
      }
#pragma unroll
      for (int u = 0; u < V; ++u) y.v[u] *= f1;
      if (two) {
        Pack<V> z = y2(i);
        if (a.y2_norm) {
          const Pack<V> w = ld_bf16<V>(a.y2_norm + i);
#pragma unroll
          for (int u = 0; u < V; ++u) z.v[u] *= w.v[u];
        }
#pragma unroll
        for (int u = 0; u < V; ++u) y.v[u] = fmaf(f2, z.v[u], y.v[u]);
      }
      Pack<V> nx[S];
#pragma unroll
      for (int t = 0; t < S; ++t) {
#pragma unroll
        for (int u = 0; u < V; ++u) {
          float v = outv[t] * y.v[u];
#pragma unroll
          for (int s = 0; s < S; ++s) v = fmaf(mix[s * S + t], x[s].v[u], v);
          nx[t].v[u] = v;
        }
      }
#pragma unroll
      for (int t = 0; t < S; ++t) {
        x[t] = nx[t];
        st_f32<V>(Xr + (size_t)t * W + i, nx[t]);
      }
      if (a.dump) {
        Pack<V> d;
#pragma unroll
        for (int u = 0; u < V; ++u) {
          d.v[u] = x[0].v[u];
#pragma unroll
          for (int s = 1; s < S; ++s) d.v[u] += x[s].v[u];
        }
        st_f32<V>(a.dump + (size_t)r * W + i, d);
      }
    }
    if (read || a.sum_out) {
      Pack<V> p;
#pragma unroll
      for (int u = 0; u < V; ++u) {
        float v = 0.f;
#pragma unroll
        for (int s = 0; s < S; ++s) v = fmaf(inv[s], x[s].v[u], v);
        p.v[u] = v;
        sum = a.b ? sum + v : fmaf(v, v, sum);
      }
      if (a.sum_out) st_f32<V>(a.sum_out + (size_t)r * W + i, p);
      if (read) {
        if (a.w) {
          st_f32<V>(row + i, p);  // normed below
        } else {
          if (a.h) st_f32<V>(a.h + (size_t)r * W + i, p);
          if (a.h_bf) st_bf16<V>(a.h_bf + (size_t)r * W + i, p);
        }
      }
    }
  }
  if (!read || !a.w) return;
  float mean = 0.f, var = block_sum_r(sum, red) / (float)W;
  if (a.b) {  // layer norm: the mean comes off first; every thread rereads only what it wrote
    mean = var;
    float q = 0.f;
    for (int i = t0; i < W; i += step) {
      const Pack<V> p = ld_f32<V>(row + i);
#pragma unroll
      for (int u = 0; u < V; ++u) q = fmaf(p.v[u] - mean, p.v[u] - mean, q);
    }
    var = block_sum_r(q, red) / (float)W;
  }
  const float rstd = 1.0f / sqrtf(var + a.eps);
  for (int i = t0; i < W; i += step) {
    Pack<V> p = ld_f32<V>(row + i);
    const Pack<V> w = ld_bf16<V>(a.w + i);
#pragma unroll
    for (int u = 0; u < V; ++u) p.v[u] = (p.v[u] - mean) * rstd * w.v[u];
    if (a.b) {
      const Pack<V> b = ld_bf16<V>(a.b + i);
#pragma unroll
      for (int u = 0; u < V; ++u) p.v[u] += b.v[u];
    }
    if (a.h) st_f32<V>(a.h + (size_t)r * W + i, p);
    if (a.h_bf) st_bf16<V>(a.h_bf + (size_t)r * W + i, p);
  }
}

template <int V>
cudaError_t launch_hyper_v(const HyperStep& a, size_t smem, cudaStream_t st) {
  void (*kern)(const HyperStep) = nullptr;
  switch (a.streams) {
    case 1: kern = hyper_step_kernel<1, V>; break;
    case 2: kern = hyper_step_kernel<2, V>; break;
    case 3: kern = hyper_step_kernel<3, V>; break;
    case 4: kern = hyper_step_kernel<4, V>; break;
    case 5: kern = hyper_step_kernel<5, V>; break;
    case 6: kern = hyper_step_kernel<6, V>; break;
    case 7: kern = hyper_step_kernel<7, V>; break;
    default: kern = hyper_step_kernel<8, V>; break;
  }
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) return cudaErrorInvalidValue;
    cudaError_t r = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (r != cudaSuccess) return r;
  }
  return launch_k(kern, dim3(a.n), dim3(256), smem, st, a);
}

}  // namespace

cudaError_t launch_embed_streams(float* X, const bf16* embed, const bf16* pos_table, const int* ids, const int* pos, int width, int streams,
                                 int n, cudaStream_t st) {
  if (n <= 0) return cudaSuccess;
  return launch_k(embed_streams_kernel, dim3(n), dim3(width >= 1024 ? 256 : 128), 0, st, X, embed, pos_table, ids, pos, width, streams);
}

cudaError_t launch_hyper_step(const HyperStep& a, cudaStream_t st) {
  if (a.n <= 0) return cudaSuccess;
  if (a.streams < 1 || a.streams > HC_MAX_STREAMS) return cudaErrorInvalidValue;
  const bool write = a.y1 || a.y1_bf;
  if ((write && (a.gather || a.ids)) || (a.ids && (!a.embed || a.gather)) || (a.b && !a.w) || (a.y2_norm && !a.y1_norm)) return cudaErrorInvalidValue;
  const size_t smem = a.w && (a.h || a.h_bf) ? (size_t)a.width * sizeof(float) : 0;
  auto al = [](const void* p, size_t b) { return (reinterpret_cast<uintptr_t>(p) & (b - 1)) == 0; };
  const bool vec = a.width % 4 == 0 && al(a.X, 16) && al(a.y1, 16) && al(a.y2, 16) && al(a.y1_bf, 8) && al(a.y2_bf, 8) && al(a.y1_norm, 8) &&
                   al(a.y2_norm, 8) && al(a.embed, 8) && al(a.w, 8) && al(a.b, 8) && al(a.h, 16) && al(a.h_bf, 8) && al(a.sum_out, 16) && al(a.dump, 16);
  return vec ? launch_hyper_v<4>(a, smem, st) : launch_hyper_v<1>(a, smem, st);
}

}  // namespace qie
