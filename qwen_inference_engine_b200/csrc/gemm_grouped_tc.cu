// gemm_grouped_tc.cu -- the expert GEMMs of a mixture of experts on the 5th-gen tensor cores (nogatar.h: GroupedGemmBf16): rows grouped by
// expert, one weight matrix [N, K] per expert.  A persistent CTA per SM walks tiles of 128 rows of one expert x 256 weight rows;
// which tiles there are stands in grp_off on the device.  10 warps:
//   warp 0     operand tiles by TMA into a ring of four stages (64 k-elements each)
//   warp 1     D[row, weight row] += A W^T: tcgen05.mma 128 x 256 x 16, two accumulators of 256 TMEM columns
//   warps 2-9  epilogue of the tile before: a thread holds a row; in the gated mode its tile is [128 gate | 128 up] rows of the same
//              columns, so that silu's argument and its factor meet in one thread and only silu(gate) * up goes to memory
// Rows behind a group's last (the next group's, or zeros) are multiplied and dropped.  k ascends per output whatever the tile, so a
// row's result does not depend on the rows around it.  Gathered rows (row_idx) are brought in order by a kernel in front.
// Every wait has a limit; when one runs out the CTA finishes without waiting and marks its results as not a number.
#include <cuda.h>

#include <algorithm>

#include "kernels.h"
#include "launch.h"
#include "nogatar.h"
#include "tc_ptx.cuh"

namespace qie {
namespace {

constexpr int GM = 128, GN = 256, GK = 64, GS = 4;
constexpr int A_BYTES = GM * GK * 2, B_BYTES = GN * GK * 2, STAGE = A_BYTES + B_BYTES;
constexpr int GTHREADS = 320;
constexpr int MAX_GROUPS = 1024;
constexpr size_t GSMEM = (size_t)GS * STAGE + 1024 /*align*/ + 256 /*barriers*/;

__device__ __forceinline__ void tma_2d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int c0, int c1) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
      ::"r"(dst), "l"(map), "r"(bar), "r"(c0), "r"(c1)
      : "memory");
}

// silu(z) for a result that is rounded to bf16
__device__ __forceinline__ float silu_short(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

__global__ void __launch_bounds__(GTHREADS, 1) grouped_gemm_tc_kernel(const GroupedGemmBf16 g, const __grid_constant__ CUtensorMap map_a,
                                                                      const __grid_constant__ CUtensorMap map_w, int n_tiles) {
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  __shared__ int tile0[MAX_GROUPS + 1];  // row tiles in front of every group
  __shared__ int dead_s;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t s0 = (smem_u32(smem_raw) + 1023u) & ~1023u, bars = s0 + GS * STAGE;
  auto full = [&](uint32_t s) { return bars + 8 * s; };
  auto empty = [&](uint32_t s) { return bars + 8 * (GS + s); };
  auto ready = [&](uint32_t b) { return bars + 8 * (2 * GS + b); };      // accumulator b is complete
  auto drained = [&](uint32_t b) { return bars + 8 * (2 * GS + 2 + b); };  // accumulator b may be overwritten
  const uint32_t tslot = bars + 8 * (2 * GS + 4);
  volatile int* dead = &dead_s;
  if (tid == 0) {
    dead_s = 0;
    for (int s = 0; s < GS; ++s) mbar_init_tc(full(s), 1), mbar_init_tc(empty(s), 1);
    for (int b = 0; b < 2; ++b) mbar_init_tc(ready(b), 1), mbar_init_tc(drained(b), GTHREADS - 64);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tslot), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  pdl_wait();
  pdl_trigger();
  if (warp == 2) {  // row tiles per group, summed up
    int run = 0;
    for (int z0 = 0; z0 < g.groups; z0 += 32) {
      const int z = z0 + lane, cnt = z < g.groups ? (g.grp_off[z + 1] - g.grp_off[z] + GM - 1) / GM : 0;
      int inc = cnt;
      for (int o = 1; o < 32; o <<= 1) {
        const int t = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= o) inc += t;
      }
      if (z < g.groups) tile0[z + 1] = run + inc;
      run += __shfl_sync(0xffffffffu, inc, 31);
    }
    if (lane == 0) tile0[0] = 0;
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  uint32_t tmem;
  asm volatile("ld.shared.b32 %0, [%1];" : "=r"(tmem) : "r"(tslot));
  const int total = tile0[g.groups] * n_tiles, nkb = (g.K + GK - 1) / GK;
  const int n_out = g.gated ? g.N / 2 : g.N, per = g.gated ? GN / 2 : GN;  // output columns in all and per tile

  if (warp == 0) {
    if (lane == 0) {
      uint32_t it = 0;
      int z = 0;
      for (int t = blockIdx.x; t < total && !*dead; t += gridDim.x) {
        const int rt = t / n_tiles, c0 = (t - rt * n_tiles) * per;
        while (rt >= tile0[z + 1]) ++z;
        const int a_row = g.grp_off[z] + (rt - tile0[z]) * GM;
        const int w0 = z * g.N + c0, w1 = g.gated ? w0 + n_out : w0 + GN / 2;
        for (int kb = 0; kb < nkb; ++kb, ++it) {
          const uint32_t s = it % GS, sa = s0 + s * STAGE;
          mbar_wait_tc(empty(s), ((it / GS) & 1) ^ 1, dead);
          if (*dead) break;
          asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(full(s)), "r"((uint32_t)STAGE) : "memory");
          tma_2d(sa, &map_a, full(s), kb * GK, a_row);
          tma_2d(sa + A_BYTES, &map_w, full(s), kb * GK, w0);
          tma_2d(sa + A_BYTES + B_BYTES / 2, &map_w, full(s), kb * GK, w1);
        }
      }
      if (*dead)  // copies may still be in flight: give them time to land
        for (const long long c = clock64(); clock64() - c < 2000000;) {
        }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = idesc_tc(GM, GN, false);
      uint32_t it = 0, j = 0;
      for (int t = blockIdx.x; t < total && !*dead; t += gridDim.x, ++j) {
        const uint32_t b = j & 1;
        mbar_wait_tc(drained(b), ((j >> 1) & 1) ^ 1, dead);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        for (int kb = 0; kb < nkb; ++kb, ++it) {
          const uint32_t s = it % GS, sa = s0 + s * STAGE, sb = sa + A_BYTES;
          mbar_wait_tc(full(s), (it / GS) & 1, dead);
          if (*dead) break;
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
          for (int k = 0; k < GK / 16; ++k) umma_tc(tmem + b * GN, desc_k_tc(sa + k * 32), desc_k_tc(sb + k * 32), idesc, (kb | k) != 0);
          umma_commit_tc(empty(s));
        }
        umma_commit_tc(ready(b));
      }
    }
    __syncwarp();
  } else {
    const int qd = warp & 3, half = (warp - 2) >> 2;  // TMEM lanes 32 qd .., half of the tile's output columns
    uint32_t j = 0;
    int z = 0;
    for (int t = blockIdx.x; t < total && !__any_sync(0xffffffffu, *dead); t += gridDim.x, ++j) {
      const uint32_t b = j & 1;
      const int rt = t / n_tiles, c0 = (t - rt * n_tiles) * per + half * (per / 2);
      while (rt >= tile0[z + 1]) ++z;
      const int m = (rt - tile0[z]) * GM + qd * 32 + lane, row_base = g.grp_off[z];
      const bool live = m < g.grp_off[z + 1] - row_base;
      const size_t row = (size_t)row_base + m;
      float rw = live && g.row_w ? g.row_w[row] : 1.f;
      mbar_wait_tc(ready(b), (j >> 1) & 1, dead);
      __syncwarp();
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      if (*dead) rw = __int_as_float(0x7fffffff);
      const uint32_t acc = tmem + b * GN + ((uint32_t)(qd * 32) << 16) + (uint32_t)(half * (per / 2));
      bf16* out = g.out_bf + row * g.ldo;
#pragma unroll 2
      for (int c = 0; c < per / 2; c += 16) {
        uint32_t r[16], u[16];
        tmem_ld16_tc(acc + c, r);
        if (g.gated) tmem_ld16_tc(acc + GN / 2 + c, u);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        float v[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          v[e] = __uint_as_float(r[e]) * rw;
          if (g.gated) v[e] = silu_short(v[e]) * (__uint_as_float(u[e]) * rw);
        }
#pragma unroll
        for (int h = 0; h < 16; h += 8)
          if (live && c0 + c + h < n_out)
            *reinterpret_cast<uint4*>(out + c0 + c + h) =
                make_uint4(pack2f(v[h], v[h + 1]), pack2f(v[h + 2], v[h + 3]), pack2f(v[h + 4], v[h + 5]), pack2f(v[h + 6], v[h + 7]));
      }
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive_tc(drained(b));
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
  }
}

// out[r, :] = in[row_idx[r], :], a warp per row, 16-byte pieces
__global__ void __launch_bounds__(256) gather_rows_bf16_kernel(const bf16* __restrict__ in, int ld, const int* __restrict__ row_idx, bf16* __restrict__ out,
                                                               int cols, int n) {
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= n) return;
  const uint4* src = reinterpret_cast<const uint4*>(in + (size_t)row_idx[r] * ld);
  uint4* dst = reinterpret_cast<uint4*>(out + (size_t)r * cols);
#pragma unroll 4
  for (int i = lane; i < cols / 8; i += 32) dst[i] = src[i];
}

}  // namespace

bool grouped_gemm_tc_fits(const GroupedGemmBf16& g) {
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return g.out_bf && g.K >= 128 && g.K % 8 == 0 && g.N >= 128 && g.N % 16 == 0 && g.w_batch == (long)g.N * g.K && g.groups <= MAX_GROUPS && g.ldo % 8 == 0 &&
         g.lda % 8 == 0 && (g.row_idx ? g.a_rows != nullptr : g.lda == g.K) && (long)g.groups * g.N < (1l << 31) && al(g.A) && al(g.W) && al(g.out_bf) && al(g.a_rows);
}

cudaError_t launch_grouped_gemm_tc(const GroupedGemmBf16& g, int num_sms, cudaStream_t st) {
  cudaError_t r;
  static PerDeviceOnce set;
  if (set.need()) {
    if ((r = cudaFuncSetAttribute(grouped_gemm_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)GSMEM)) != cudaSuccess) return r;
    set.done();
  }
  if (g.row_idx && (r = launch_k(gather_rows_bf16_kernel, dim3((g.rows + 7) / 8), dim3(256), 0, st, g.A, g.lda, g.row_idx, g.a_rows, g.K, g.rows)) != cudaSuccess)
    return r;
  TensorMap2D ma{}, mw{};
  if ((r = make_tensor_map_2d(&ma, g.row_idx ? g.a_rows : g.A, g.rows, g.K, GM)) != cudaSuccess) return r;
  if ((r = make_tensor_map_2d(&mw, g.W, g.groups * g.N, g.K, GN / 2)) != cudaSuccess) return r;
  const int n_out = g.gated ? g.N / 2 : g.N, per = g.gated ? GN / 2 : GN, n_tiles = (n_out + per - 1) / per;
  const int most = (g.rows / GM + std::min(g.rows, g.groups)) * n_tiles;  // an upper bound of the tiles
  return launch_k(grouped_gemm_tc_kernel, dim3(std::min(num_sms, most)), dim3(GTHREADS), GSMEM, st, g, *reinterpret_cast<const CUtensorMap*>(&ma),
                  *reinterpret_cast<const CUtensorMap*>(&mw), n_tiles);
}

}  // namespace qie
