// attn_gqa_tc.cu -- prompt attention over paged bf16 key/value rows on the 5th-gen tensor cores (tcgen05 + TMEM), for grouped
// queries under a sliding window, a causal mask or chunks of positions, and pooled rows.  A plain head attends to the values of its kv
// head and writes its output rows.  The softmax weights may be mixed over the heads (GqaAttnArgs::talk).  Mixing after the softmax is linear, so every head attends to the values of ALL kv heads -- one product with up to
// 256 value columns, which is what the tensor cores are good at -- and gqa_talk_mix_kernel mixes the results.
//
// A CTA owns 128 consecutive rows of one segment, one query head and one chunk of value columns, and walks tiles of 64 keys: first
// the tiles of pooled rows that some row sees, then the tokens from the first window's lower edge on.  20 warps:
//   the last 3  bring the tile's key and value rows into the swizzled operand layout, a ring of stages: token rows by TMA boxes of
//               a page, pooled rows (and token rows of pages that do not divide a tile) by cp.async; the first pooled tiles are
//               copied by all warps before they take their roles
//   warp 16     issues the products: S = Q K^T (128 x 64, two TMEM buffers, one tile ahead of the softmax) and O += P V
//   warps 0-15  softmax, four threads per row: S from TMEM, mask, reference maximum, weights as bf16 hi + lo pairs into TMEM (two
//               buffers; the second product takes its A operand from there), two products per tile, so a weight keeps ~16 bits
// O stays in TMEM over all tiles.  Instead of scaling it whenever a row's maximum grows, a row keeps its reference maximum until a
// score exceeds it by RESCALE (weights then stay below 2^RESCALE); only then the warp that owns the row scales its part of O.
// Every wait has a limit; when one runs out the CTA finishes without waiting and marks its results as not a number.
#include <cuda.h>

#include <algorithm>

#include "common.cuh"
#include "fosavik.h"
#include "kernels.h"
#include "kv_rows.cuh"
#include "launch.h"
#include "tc_ptx.cuh"

namespace qie {
namespace {

constexpr int TQ = 128, TK = 64;
constexpr int NSOFT = 512, NLOAD = 96, MMA_WARP = NSOFT / 32, NTHR = NSOFT + 32 + NLOAD;
constexpr int LROWS = NLOAD / 8, LPASS = (TK + LROWS - 1) / LROWS;  // rows a pass of the copying threads covers
constexpr int MAX_ST = 6, TURN = 33;                                // stages at most; row pitch of the turned results
constexpr int KBLK = TK * 128;   // [64 keys][64 columns] bf16, 8-row swizzle atoms: 8 KiB
constexpr int QBLK = TQ * 128;   // [128 rows][64 columns]: 16 KiB
constexpr float RESCALE = 8.0f;  // in powers of two

// byte offset of 16-byte chunk ch (0..7) of row r in a block of 64 columns
__device__ __forceinline__ uint32_t blk_off(int r, int ch) { return (uint32_t)(r * 128 + ((ch ^ (r & 7)) << 4)); }

struct TcLayout {  // byte offsets from the 1024-aligned base
  int dblk, vblk, nst, q, st, stage, bar, total;
};
__host__ __device__ inline TcLayout tc_layout(int dblk, int vblk, int nst) {
  TcLayout l;
  l.dblk = dblk, l.vblk = vblk, l.nst = nst;
  l.q = 0;
  l.st = l.q + dblk * QBLK;       // stages: K blocks | V blocks; at the end the results are turned around there
  l.stage = (dblk + vblk) * KBLK;
  l.bar = l.st + (nst * l.stage > NSOFT * TURN * 4 ? nst * l.stage : (NSOFT * TURN * 4 + 1023) / 1024 * 1024);  // mbarriers, flags, row maxima
  l.total = l.bar + 256 + 8 * TQ * 4;
  return l;
}

// chunk ch (16 bytes) of every 64-column block of one key row and its values -> row r of the stage at `base`; null: zeros
__device__ __forceinline__ void copy_row(const bf16* row, size_t koff, size_t voff, uint32_t base, int r, int ch, int dblk, int vblk, int dim, int nv) {
  for (int b = 0; b < dblk + vblk; ++b) {
    const bool isv = b >= dblk;
    const int c = (isv ? b - dblk : b) * 64 + ch * 8;
    const uint32_t dst = base + b * KBLK + blk_off(r, ch);
    if (row && c < (isv ? nv : dim)) cp_async16(dst, row + (isv ? voff : koff) + c);
    else asm volatile("st.shared.v4.b32 [%0], {%1,%1,%1,%1};" ::"r"(dst), "r"(0u) : "memory");
  }
}

// Tiles of a segment in ascending order of how deep in its chunk a tile lies, which is how many keys it sees: number i of nt.  m tiles make
// about one chunk; a tile's depth is its number modulo m, counted from where the segment's first row (position p0) lies in its chunk.
__device__ __forceinline__ int by_work(int i, int nt, int p0, int chunk) {
  const int m = min((chunk + TQ - 1) / TQ, nt), off = p0 % chunk / TQ % m;
  for (int r = 0; r < m; ++r) {
    const int first = (r - off + m) % m, count = first < nt ? (nt - first + m - 1) / m : 0;
    if (i < count) return first + i * m;
    i -= count;
  }
  return 0;  // not reached: the counts add up to nt
}

__global__ void __launch_bounds__(NTHR, 1) gqa_tc_kernel(const GqaAttnArgs a, int dblk, int vblk, int nst, int vc,
                                                               const __grid_constant__ CUtensorMap rows_map, int use_tma) {
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  __shared__ int info[4];  // first row, rows, slot
  __shared__ int dead_s;
  pdl_wait();
  pdl_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    int left = gridDim.y - 1 - blockIdx.y, found = 0;  // late tiles of a segment see more keys: they start first
    for (int s = 0; s < a.n_seg && !found; ++s) {
      const int r0 = a.seg_start[s], len = a.seg_start[s + 1] - r0, nt = (len + TQ - 1) / TQ;
      if (left >= 0 && left < nt) {
        const int t = a.chunk > 0 ? by_work(left, nt, a.pos[r0], a.chunk) : left;
        info[0] = r0 + t * TQ, info[1] = min(TQ, len - t * TQ), info[2] = a.seg_slot[s], found = 1;
      }
      left -= nt;
    }
    if (!found) info[1] = 0;
    dead_s = 0;
  }
  __syncthreads();
  const int row0 = info[0], nrows = info[1], slot = info[2];
  if (nrows == 0) return;
  volatile int* dead = &dead_s;
  const TcLayout L = tc_layout(dblk, vblk, nst);
  const uint32_t s0 = (smem_u32(smem_raw) + 1023u) & ~1023u;
  unsigned char* sg = smem_raw + (s0 - smem_u32(smem_raw));
  const uint32_t b0 = s0 + L.bar;
  const uint32_t bar_full = b0, bar_empty = b0 + 8 * MAX_ST, bar_s = b0 + 16 * MAX_ST, bar_p = bar_s + 16, bar_o = bar_s + 32, tslot = bar_s + 48;
  float* xmax = reinterpret_cast<float*>(sg + L.bar + 256);  // [tile parity][quarter][row]; the sums use the parity that the last tile did not
  const int h = blockIdx.x, g = h / (a.heads / a.kv_heads), dim = a.dim;
  // value columns: chunk blockIdx.z of those of all kv heads, or (plain heads) the columns of head h's kv head
  const int vcols = a.talk ? a.kv_heads * a.vdim : a.vdim, zc = blockIdx.z * vc, nv = min(vc, vcols - zc), col0 = a.talk ? zc : g * a.vdim + zc;
  const int pos0 = a.pos[row0], pmax = pos0 + nrows - 1;
  const int lo_min = first_seen(pos0, a.window, a.chunk);
  const int nbmax = a.c.block > 0 ? pooled_seen(pmax, a.window, a.c.block) : 0, npt = (nbmax + TK - 1) / TK;
  const int tt0 = lo_min / TK, nt = npt + pmax / TK - tt0 + 1;  // tiles: npt of pooled rows, then tokens from tile tt0 on
  if (tid == 0) {
    for (int i = 0; i < nst; ++i) mbar_init_tc(bar_full + 8 * i, NLOAD / 32), mbar_init_tc(bar_empty + 8 * i, 1);
    for (int i = 0; i < 2; ++i) mbar_init_tc(bar_s + 8 * i, 1), mbar_init_tc(bar_p + 8 * i, NSOFT), mbar_init_tc(bar_o + 8 * i, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == MMA_WARP) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tslot), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  // the first tiles of pooled rows, as many as there are stages: thread = (row, 16-byte chunk of a block)
  const int npre = min(npt, nst);
  const size_t koff = (size_t)g * dim, voff = (size_t)a.c.kw + col0;
  for (int t = 0; t < npre; ++t) {
    const int r = tid >> 3, ch = tid & 7, b = t * TK + r;
    if (r >= TK) break;
    const bf16* row = b < nbmax ? reinterpret_cast<const bf16*>(kv_pool_ptr(a.c, a.block_table, a.max_pages, slot, b)) : nullptr;
    copy_row(row, koff, voff, s0 + L.st + t * L.stage, r, ch, dblk, vblk, dim, nv);
  }
  cp_async_commit();
  // Q rows as bf16, zeros beyond the head size and the last row (dim is a multiple of 8)
  const bool q16 = a.ldq % 4 == 0 && (reinterpret_cast<uintptr_t>(a.q) & 15) == 0;
  for (int i = tid; i < TQ * dblk * 8; i += NTHR) {
    const int r = i / (dblk * 8), c = (i - r * dblk * 8) * 8;
    uint4 w = make_uint4(0u, 0u, 0u, 0u);
    if (r < nrows && c < dim) {
      const float* q = a.q + (size_t)(row0 + r) * a.ldq + (size_t)h * dim + c;
      if (q16) {
        const float4 x = *reinterpret_cast<const float4*>(q), y = *reinterpret_cast<const float4*>(q + 4);
        w = make_uint4(pack2f(x.x, x.y), pack2f(x.z, x.w), pack2f(y.x, y.y), pack2f(y.z, y.w));
      } else {
        w = make_uint4(pack2f(q[0], q[1]), pack2f(q[2], q[3]), pack2f(q[4], q[5]), pack2f(q[6], q[7]));
      }
    }
    *reinterpret_cast<uint4*>(sg + L.q + (c >> 6) * QBLK + blk_off(r, (c >> 3) & 7)) = w;
  }
  cp_async_wait<0>();
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  uint32_t tmem;
  asm volatile("ld.shared.b32 %0, [%1];" : "=r"(tmem) : "r"(tslot));
  const uint32_t t_o = tmem + 128, t_p = tmem + 384;  // S: columns 0..127 (two buffers), O: 128 .. 383, P: 384 .. (two buffers of hi | lo)
  const int vcp = vblk * 64;        // columns of O

  if (warp > MMA_WARP) {
    // ---- copies
    const int lt = tid - (NSOFT + 32), lw = warp - MMA_WARP - 1, ch = lt & 7, rr = lt >> 3;  // cp.async: chunk of a block, rows rr + LROWS k
    // TMA: boxes of up to 64 rows of a page and 64 columns, box number 3 * lane + lw.  Rows behind the last position and columns behind
    // a part are other cache contents: finite numbers that meet zero weights, zero queries or columns nobody reads.
    const int br = min(a.c.page_size, TK), nbx = TK / br, boxes = nbx * (dblk + vblk), bi = 3 * lane + lw, bb = bi / nbx, pg = bi - bb * nbx;
    const int bx = bb < dblk ? g * dim + bb * 64 : a.c.kw + col0 + (bb - dblk) * 64;
    const uint32_t bdst = (uint32_t)(bb * KBLK + pg * br * 128), wbytes = (uint32_t)((boxes - lw + 2) / 3 * br * 128);
    const int* bt = a.block_table + (size_t)slot * a.max_pages;
    auto page_of = [&](int t) { return bt[min((tt0 + t - npt) * TK + pg * br, pmax) / a.c.page_size]; };
    auto announce = [&](int t) {  // the copies of tile t are complete: visible to the tensor core
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive_tc(bar_full + 8 * (t % nst));
    };
    int page = use_tma && bi < boxes && npt < nt ? page_of(npt) : 0;
    bool prev_cp = false;  // the tile before was copied by cp.async and is not announced yet
    for (int t = 0; t < nt; ++t) {
      const int s = t % nst;
      if (t < npre) {  // copied above
        if (lane == 0) mbar_arrive_tc(bar_full + 8 * s);
        continue;
      }
      const bool tma = use_tma && t >= npt;
      if (prev_cp && (nst == 2 || tma)) {  // (two stages: the stage that this tile waits for is only given back behind the scores of the tile before)
        cp_async_wait<0>();
        announce(t - 1);
        prev_cp = false;
      }
      if (t >= nst) mbar_wait_tc(bar_empty + 8 * s, (uint32_t)((t / nst - 1) & 1), dead);
      const uint32_t base = s0 + L.st + s * L.stage;
      if (tma) {
        if (lane == 0) asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar_full + 8 * s), "r"(wbytes) : "memory");
        __syncwarp();
        if (bi < boxes) {
          asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
                       ::"r"(base + bdst), "l"(&rows_map), "r"(bar_full + 8 * s), "r"(bx), "r"((tt0 + t - npt) * TK % a.c.page_size), "r"(page)
                       : "memory");
          if (t + 1 < nt) page = page_of(t + 1);
        }
        continue;
      }
      const bf16* rowp[LPASS];
#pragma unroll
      for (int k = 0; k < LPASS; ++k) {
        const int r = rr + LROWS * k;
        const char* p = nullptr;
        if (t < npt) {
          if (r < TK && t * TK + r < nbmax) p = kv_pool_ptr(a.c, a.block_table, a.max_pages, slot, t * TK + r);
        } else {
          const int j = (tt0 + t - npt) * TK + r;
          if (r < TK && j <= pmax) p = kv_row_ptr(a.c, a.block_table, a.max_pages, slot, j);
        }
        rowp[k] = reinterpret_cast<const bf16*>(p);
      }
#pragma unroll
      for (int k = 0; k < LPASS; ++k)
        if (rr + LROWS * k < TK) copy_row(rowp[k], koff, voff, base, rr + LROWS * k, ch, dblk, vblk, dim, nv);
      cp_async_commit();
      if (prev_cp) {
        cp_async_wait<1>();
        announce(t - 1);
      }
      prev_cp = true;
    }
    if (prev_cp) {
      cp_async_wait<0>();
      announce(nt - 1);
    }
  } else if (warp == MMA_WARP) {
    // ---- products
    if (lane == 0) {
      const uint32_t id_s = idesc_tc(TQ, TK, false), id_o = idesc_tc(TQ, vcp, true);
      auto issue_s = [&](int t) {
        const int s = t % nst;
        mbar_wait_tc(bar_full + 8 * s, (uint32_t)((t / nst) & 1), dead);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t kb = s0 + L.st + s * L.stage;
        for (int kk = 0; kk < dblk * 4; ++kk)
          umma_tc(tmem + (uint32_t)((t & 1) * TK), desc_k_tc(s0 + L.q + (kk >> 2) * QBLK + (kk & 3) * 32), desc_k_tc(kb + (kk >> 2) * KBLK + (kk & 3) * 32),
                  id_s, kk != 0);
        umma_commit_tc(bar_s + 8 * (t & 1));
      };
      issue_s(0);
      for (int t = 0; t < nt; ++t) {
        if (t + 1 < nt) issue_s(t + 1);  // its buffer was read before the weights of tile t - 1 were announced
        mbar_wait_tc(bar_p + 8 * (t & 1), (uint32_t)((t >> 1) & 1), dead);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t vb = s0 + L.st + (t % nst) * L.stage + dblk * KBLK, ph = t_p + (uint32_t)((t & 1) * TK);
        for (int part = 0; part < 2; ++part)  // hi, lo
          for (int kk = 0; kk < TK / 16; ++kk)
            umma_ts_tc(t_o, ph + (uint32_t)(part * (TK / 2) + kk * 8), desc_mn_tc(vb + kk * 16 * 128, KBLK), id_o, t > 0 || part > 0 || kk > 0);
        umma_commit_tc(bar_empty + 8 * (t % nst));
        umma_commit_tc(bar_o + 8 * (t & 1));
      }
    }
    __syncwarp();
  } else {
    // ---- softmax: row (TMEM lane), quarter of the tile's keys and of O's columns
    const int row = (warp & 3) * 32 + lane, qt = warp >> 2;
    const int my_pos = pos0 + row, my_lo = first_seen(my_pos, a.window, a.chunk), my_seen = a.c.block > 0 ? pooled_seen(my_pos, a.window, a.c.block) : 0;
    const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;
    const float sl2 = a.scale * 1.4426950408889634f;
    const int oc0 = qt * (vcp / 4), oc1 = oc0 + vcp / 4;
    float m_ref = -INFINITY, l_run = 0.f;
    for (int t = 0; t < nt; ++t) {
      mbar_wait_tc(bar_s + 8 * (t & 1), (uint32_t)((t >> 1) & 1), dead);
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      uint32_t r[16];
      tmem_ld16_tc(tmem + lane_addr + (uint32_t)((t & 1) * TK + 16 * qt), r);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      // visible keys of this thread: first .. last (relative to its 16)
      int first, last;
      if (t < npt) first = 0, last = my_seen - 1 - (t * TK + 16 * qt);
      else first = my_lo - ((tt0 + t - npt) * TK + 16 * qt), last = my_pos - ((tt0 + t - npt) * TK + 16 * qt);
      if (first > 0 || last < 15) {
#pragma unroll
        for (int j = 0; j < 16; ++j)
          if (j < first || j > last) r[j] = 0xff800000u;  // -inf
      }
      float mx = -INFINITY;
#pragma unroll
      for (int j = 0; j < 16; ++j) mx = fmaxf(mx, __uint_as_float(r[j]));
      float* xm = xmax + (t & 1) * 4 * TQ + row;
      xm[qt * TQ] = mx;
      asm volatile("bar.sync %0, 128;" ::"r"(1 + (warp & 3)) : "memory");  // the four warps that share these 32 rows
      mx = fmaxf(fmaxf(xm[0], xm[TQ]), fmaxf(xm[2 * TQ], xm[3 * TQ])) * sl2;
      const bool grow = mx > m_ref + RESCALE;
      if (__any_sync(0xffffffffu, grow)) {
        const float m_new = fmaxf(m_ref, mx), f = m_new > -INFINITY ? ex2_tc(m_ref - m_new) : 1.f;
        m_ref = m_new, l_run *= f;
        if (t > 0) {  // scale this thread's columns of O once the product of the tile before is in
          mbar_wait_tc(bar_o + 8 * ((t - 1) & 1), (uint32_t)(((t - 1) >> 1) & 1), dead);
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          for (int c = oc0; c < oc1; c += 16) {
            uint32_t o[16];
            tmem_ld16_tc(t_o + lane_addr + c, o);
            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
            for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * f);
            tmem_st16_tc(t_o + lane_addr + c, o);
          }
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
      }
      const float nm = m_ref > -INFINITY ? -m_ref : 0.f;
      float rs = 0.f;
      uint32_t hi[8], lo[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float e0 = ex2_tc(fmaf(__uint_as_float(r[2 * e]), sl2, nm)), e1 = ex2_tc(fmaf(__uint_as_float(r[2 * e + 1]), sl2, nm));
        rs += e0 + e1;
        hi[e] = pack2f(e0, e1);
        lo[e] = pack2f(e0 - lo2f(hi[e]), e1 - hi2f(hi[e]));
      }
      l_run += rs;
      if (t >= 2) mbar_wait_tc(bar_o + 8 * (t & 1), (uint32_t)(((t >> 1) - 1) & 1), dead);  // the product that read this P buffer
      const uint32_t pd = t_p + lane_addr + (uint32_t)((t & 1) * TK + 8 * qt);
      tmem_st8_tc(pd, hi);
      tmem_st8_tc(pd + TK / 2, lo);
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive_tc(bar_p + 8 * (t & 1));
    }
    mbar_wait_tc(bar_o + 8 * ((nt - 1) & 1), (uint32_t)(((nt - 1) >> 1) & 1), dead);
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    float* xs = xmax + (nt & 1) * 4 * TQ + row;
    xs[qt * TQ] = l_run;
    asm volatile("bar.sync %0, 128;" ::"r"(1 + (warp & 3)) : "memory");
    const float l = (xs[0] + xs[TQ]) + (xs[2 * TQ] + xs[3 * TQ]);
    const float inv = *dead ? __int_as_float(0x7fffffff) : (l > 0.f ? 1.0f / l : 0.f);
    const size_t rs_rec = (size_t)vcols + 2;
    const int wrow0 = row0 + (warp & 3) * 32;
    float* rec = a.ws + ((size_t)(row0 + (warp & 3) * 32) * a.heads + h) * rs_rec;  // record of the warp's first row
    const size_t row_step = (size_t)a.heads * rs_rec;
    const int wrows = min(32, nrows - (warp & 3) * 32);
    float* tr = reinterpret_cast<float*>(sg + L.st) + warp * (32 * TURN);  // every product is done: the stages are free to turn the rows around
    for (int c = oc0; c < oc1; c += 32) {
      const int cw = min(32, oc1 - c);  // 32 or 16 columns
      uint32_t o[16];
      __syncwarp();
      for (int u = 0; u < cw; u += 16) {
        tmem_ld16_tc(t_o + lane_addr + c + u, o);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
        for (int j = 0; j < 16; ++j) tr[lane * TURN + u + j] = __uint_as_float(o[j]) * inv;
      }
      __syncwarp();
      const int x = lane & (cw - 1), cc = c + x, rstep = 32 / cw;
      if (cc >= nv) continue;
      if (a.talk) {
        for (int i = lane / cw; i < wrows; i += rstep) rec[i * row_step + 2 + col0 + cc] = tr[i * TURN + x];
      } else {
        const size_t oc = (size_t)h * a.vdim + zc + cc;
        for (int i = lane / cw; i < wrows; i += rstep) {
          if (a.out_bf) a.out_bf[(size_t)(wrow0 + i) * a.ldo_bf + oc] = f2bf(tr[i * TURN + x]);
          else a.out[(size_t)(wrow0 + i) * a.ldo + oc] = tr[i * TURN + x];
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == MMA_WARP) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
  }
}

constexpr int SMEM_MAX = 226 * 1024;
struct TcPlan {
  int dblk, vblk, nst, vc, nvc;
  size_t smem;
};
TcPlan tc_plan(const GqaAttnArgs& a) {
  TcPlan p;
  const int vcols = a.talk ? a.kv_heads * a.vdim : a.vdim;
  p.dblk = (a.dim + 63) / 64;
  p.nvc = (vcols + 255) / 256;
  p.vc = ((vcols + p.nvc - 1) / p.nvc + 7) / 8 * 8;
  p.vblk = (p.vc + 63) / 64;
  p.nst = MAX_ST;
  while (p.nst > 2 && tc_layout(p.dblk, p.vblk, p.nst).total + 1024 > SMEM_MAX) --p.nst;
  p.smem = (size_t)tc_layout(p.dblk, p.vblk, p.nst).total + 1024;
  return p;
}

}  // namespace

bool gqa_tc_fits(const GqaAttnArgs& a) {
  return a.c.elt_bytes == 2 && a.seg_start && a.n >= 128 && a.n / a.n_seg >= 64 && a.dim <= 128 && a.dim % 8 == 0 &&
         (a.talk ? a.kv_heads * a.vdim : a.vdim) % 8 == 0 && a.heads % a.kv_heads == 0 && a.finish == 0 && !a.unit_sink && a.maps == 1 && a.scale > 0.f && a.keep_first == 0 && a.softcap == 0.f && !a.slopes && !a.shared_keys && a.c.page_elems % 8 == 0 && a.c.layer_off % 8 == 0 &&
         (a.c.kw + a.c.vw) % 8 == 0 && a.c.kw % 8 == 0 && (!a.c.block || (a.c.pool_off % 8 == 0 && a.window > 0)) &&
         (reinterpret_cast<uintptr_t>(a.c.pool) & 15) == 0 && a.heads <= 65535;
}

cudaError_t launch_gqa_tc(const GqaAttnArgs& a, cudaStream_t st) {
  const TcPlan p = tc_plan(a);
  static PerDeviceOnce once;
  if (once.need()) {
    cudaError_t r = cudaFuncSetAttribute(gqa_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX);
    if (r != cudaSuccess) return r;
    once.done();
  }
  // token rows by TMA where a tile of 64 positions is whole pages or lies in one (pages of 8, 16, 32 or a multiple of 64 positions)
  TensorMap2D tm{};
  const int ps = a.c.page_size, row = a.c.kw + a.c.vw;
  const int use_tma = a.c.n_pages > 0 && row >= 64 && (ps % TK == 0 || (TK % ps == 0 && ps >= 8)) &&
                      make_tensor_map_pages(&tm, static_cast<const bf16*>(a.c.pool) + a.c.layer_off, row, ps, a.c.n_pages, a.c.page_elems,
                                            std::min(ps, TK)) == cudaSuccess;
  return launch_k(gqa_tc_kernel, dim3(a.heads, a.n / TQ + a.n_seg, p.nvc), dim3(NTHR), p.smem, st, a, p.dblk, p.vblk, p.nst, p.vc,
                  *reinterpret_cast<const CUtensorMap*>(&tm), use_tma);
}

}  // namespace qie
