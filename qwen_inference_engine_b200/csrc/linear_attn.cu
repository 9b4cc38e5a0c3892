// linear_attn.cu -- linear attention (gebadra.h): S = decay S + k v^T, o = S^T q, an fp32 matrix per head and sequence slot, with a
// fixed decay per head, or a decay per key channel that every token gates.  Two forms of the same recurrence:
//  * token by token: a CTA owns a block of 32 value columns of one head of one segment; its state columns live in registers
//    (any head size, fp32 or bf16 sources) -- decode steps, short portions and 32-bit mode;
//  * chunks of 64 rows on tensor cores (bf16 sources, prompt portions): every chunk's own contribution to the state
//    U = sum_s decay^(L-1-s) k_s v_s^T, a carry pass S <- decay^L S + U over the chunks of a segment that leaves each chunk's
//    entry state in place of its U, and the outputs o_t = decay^(t+1) S^T q_t + sum_(s<=t) decay^(t-s) (q_t . k_s) v_s.
//    Everything that is not a projection stays fp32-like on the tensor cores: decayed keys, decayed scores and the entry
//    state enter the products as bf16 hi + lo pairs (two MMAs), accumulators are fp32.
//    With gated channels the weight of (t, s) is a sum over the channels, sum_d q_td k_sd 2^(b_td - b_sd), b the running sum of the decays'
//    logarithms inside the chunk (worked out by a kernel of its own).  It factors into a decayed query and a decayed key around a
//    reference r, q 2^(b_t - r) and k 2^(r - b_s): for keys of earlier blocks of 16 rows r is b at the query block's first row, so neither
//    factor exceeds 1; inside a block r is the middle of the block's range, as long as that range is short enough for both factors
//    to stay far inside what a float holds, else the block's 136 pairs are summed up one by one.
#include <algorithm>

#include "gebadra.h"
#include "launch.h"

namespace qie {
namespace {

constexpr int LA_TOK = 8;      // tokens staged at a time (token-by-token form)
constexpr int LA_NR = 8;       // state rows per thread
constexpr int LC = LINEAR_CHUNK;

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

// log2 of the decay of channel ch (head and key channel) in row r: log2(sigmoid(z)) inv_tau, sigmoid in the form that does not overflow
__device__ __forceinline__ float log2_sigmoid_pow(float z, float inv_tau) {
  return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * (1.4426950408889634f * inv_tau);
}
__device__ __forceinline__ float gated_log2_decay(const LinearAttnArgs& a, int r, int ch) {
  const GatedDecay& g = a.gate;
  const bf16* w = g.a2 + (size_t)ch * g.rank;
  float z = bf2f(g.bias[ch]);
  if (g.low_bf) {
    const bf16* low = g.low_bf + (size_t)r * a.ld_bf;
    for (int i = 0; i < g.rank; ++i) z = fmaf(bf2f(w[i]), bf2f(low[i]), z);
  } else {
    const float* low = g.low + (size_t)r * a.ld;
    for (int i = 0; i < g.rank; ++i) z = fmaf(bf2f(w[i]), low[i], z);
  }
  return log2_sigmoid_pow(z, g.inv_tau);
}

// CTA (head, block of 32 value columns, segment); thread = (column, part of LA_NR state rows)
template <bool GATED>
__global__ void __launch_bounds__(1024) linear_scan_kernel(const LinearAttnArgs a, int parts) {
  extern __shared__ float la_smem[];  // q [LA_TOK][DP] | k [LA_TOK][DP] | v [LA_TOK][32] | partial o [LA_TOK][parts][32] | decays [LA_TOK][DP] (GATED)
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, c0 = blockIdx.y * 32, seg = blockIdx.z;
  const int dim = a.dim, vdim = a.vdim, DP = parts * LA_NR;
  float* qs = la_smem;
  float* ks = qs + LA_TOK * DP;
  float* vs = ks + LA_TOK * DP;
  float* po = vs + LA_TOK * 32;
  float* ds = po + LA_TOK * parts * 32;
  const int tid = threadIdx.x, col = tid & 31, part = tid >> 5;
  const int r0 = a.seg_start[seg], r1 = a.seg_start[seg + 1];
  const float lam = GATED ? 0.f : a.decay_pow[h * (LC + 1) + 1];
  float* st = a.state + (size_t)a.seg_slot[seg] * a.slot_stride + (size_t)h * dim * vdim;
  const bool cv = c0 + col < vdim;
  float S[LA_NR];
#pragma unroll
  for (int i = 0; i < LA_NR; ++i) {
    const int d = part * LA_NR + i;
    S[i] = cv && d < dim ? st[(size_t)d * vdim + c0 + col] : 0.f;
  }
  auto act = [&](float z) { return a.act ? silu_f(z) : z; };
  for (int t0 = r0; t0 < r1; t0 += LA_TOK) {
    const int nt = min(LA_TOK, r1 - t0);
    __syncthreads();
    for (int i = tid; i < nt * DP; i += blockDim.x) {
      const int t = i / DP, d = i - t * DP;
      float q = 0.f, k = 0.f;
      if (d < dim) {
        if (a.q_bf) {
          const size_t o = (size_t)(t0 + t) * a.ld_bf + h * dim + d;
          q = act(bf2f(a.q_bf[o])) * a.q_scale, k = act(bf2f(a.k_bf[o])) * a.k_scale;
        } else {
          const size_t o = (size_t)(t0 + t) * a.ld + h * dim + d;
          q = act(a.q[o]) * a.q_scale, k = act(a.k[o]) * a.k_scale;
        }
      }
      qs[i] = q, ks[i] = k;
      if constexpr (GATED) ds[i] = d < dim ? exp2f(gated_log2_decay(a, t0 + t, h * dim + d)) : 0.f;
    }
    for (int i = tid; i < nt * 32; i += blockDim.x) {
      const int t = i >> 5, c = c0 + (i & 31);
      float v = 0.f;
      if (c < vdim) v = act(a.v_bf ? bf2f(a.v_bf[(size_t)(t0 + t) * a.ld_bf + h * vdim + c]) : a.v[(size_t)(t0 + t) * a.ld + h * vdim + c]);
      vs[i] = v;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float v = vs[t * 32 + col];
      const float4* q4 = reinterpret_cast<const float4*>(qs + t * DP + part * LA_NR);
      const float4* k4 = reinterpret_cast<const float4*>(ks + t * DP + part * LA_NR);
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < LA_NR / 4; ++i) {
        const float4 q = q4[i], k = k4[i];
        float4 f = make_float4(lam, lam, lam, lam);
        if constexpr (GATED) f = reinterpret_cast<const float4*>(ds + t * DP + part * LA_NR)[i];
        S[4 * i] = fmaf(f.x, S[4 * i], k.x * v), o = fmaf(S[4 * i], q.x, o);
        S[4 * i + 1] = fmaf(f.y, S[4 * i + 1], k.y * v), o = fmaf(S[4 * i + 1], q.y, o);
        S[4 * i + 2] = fmaf(f.z, S[4 * i + 2], k.z * v), o = fmaf(S[4 * i + 2], q.z, o);
        S[4 * i + 3] = fmaf(f.w, S[4 * i + 3], k.w * v), o = fmaf(S[4 * i + 3], q.w, o);
      }
      po[(t * parts + part) * 32 + col] = o;
    }
    __syncthreads();
    for (int i = tid; i < nt * 32; i += blockDim.x) {
      const int t = i >> 5, c = i & 31;
      if (c0 + c >= vdim) continue;
      float o = 0.f;
      for (int p = 0; p < parts; ++p) o += po[(t * parts + p) * 32 + c];
      a.out[(size_t)(t0 + t) * a.ldo + h * vdim + c0 + c] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < LA_NR; ++i) {
    const int d = part * LA_NR + i;
    if (cv && d < dim) st[(size_t)d * vdim + c0 + col] = S[i];
  }
}

// ---------------------------------------------------------------- chunks of 64 rows on tensor cores
__device__ __forceinline__ void ldmatrix_x2_trans_la(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];\n" : "=r"(r0), "=r"(r1) : "r"(addr));
}

constexpr int LT = 256;  // threads of the chunk kernels

// which chunk: first row, rows and segment of chunk number id (false: there is no such chunk); every thread reads the same few words
__device__ __forceinline__ bool find_chunk(const LinearAttnArgs& a, int id, int* row0, int* rows) {
  for (int s = 0; s < a.n_seg; ++s) {
    const int r0 = a.seg_start[s], len = a.seg_start[s + 1] - r0, nc = (len + LC - 1) / LC;
    if (id < nc) {
      *row0 = r0 + id * LC, *rows = min(LC, len - id * LC);
      return true;
    }
    id -= nc;
  }
  return false;
}

// 64 rows x cols of a bf16 source -> registers (every load in flight at once) -> smem tile [64][P + 8], zeros beyond, silu where asked
template <int P>
struct TileRegs {
  static constexpr int N = LC * (P / 8) / LT;
  uint4 v[N];
  __device__ __forceinline__ void load(const bf16* src, int ld, int row0, int nrows, int cols) {
    const bool vec = cols % 8 == 0 && ld % 8 == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0;
#pragma unroll
    for (int k = 0; k < N; ++k) {
      const int i = threadIdx.x + k * LT, r = i / (P / 8), c = (i % (P / 8)) * 8;
      v[k] = make_uint4(0u, 0u, 0u, 0u);
      if (r >= nrows || c >= cols) continue;
      const bf16* s = src + (size_t)(row0 + r) * ld + c;
      if (vec) {
        v[k] = *reinterpret_cast<const uint4*>(s);
      } else {
        bf16 t[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) t[e] = c + e < cols ? s[e] : f2bf(0.f);
        v[k] = make_uint4(pack2(t[0], t[1]), pack2(t[2], t[3]), pack2(t[4], t[5]), pack2(t[6], t[7]));
      }
    }
  }
  __device__ __forceinline__ void store(bf16 (*dst)[P + 8], int act) {
#pragma unroll
    for (int k = 0; k < N; ++k) {
      const int i = threadIdx.x + k * LT, r = i / (P / 8), c = (i % (P / 8)) * 8;
      uint4 x = v[k];
      if (act) {
        x.x = pack2f(silu_f(lo2f(x.x)), silu_f(hi2f(x.x))), x.y = pack2f(silu_f(lo2f(x.y)), silu_f(hi2f(x.y)));
        x.z = pack2f(silu_f(lo2f(x.z)), silu_f(hi2f(x.z))), x.w = pack2f(silu_f(lo2f(x.w)), silu_f(hi2f(x.w)));
      }
      *reinterpret_cast<uint4*>(&dst[r][c]) = x;
    }
  }
};

// U = K'^T V of a chunk, K' the decayed keys as hi + lo tiles -> ws, value columns v0 ..  A warp takes 16 state rows x half of the columns.
template <int DP, int VP>
__device__ __forceinline__ void chunk_state_product(const LinearAttnArgs& a, bf16 (*Kh)[DP + 8], bf16 (*Kl)[DP + 8], bf16 (*Vs)[VP + 8], int h, int v0) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int HB = VP / 16;  // blocks of 8 columns per half
  const int dim = a.dim, vdim = min(VP, a.vdim - v0);  // value columns of this CTA
  float* U = a.ws + ((size_t)blockIdx.x * a.heads + h) * dim * a.vdim + v0;
  for (int u = warp; u < DP / 8; u += LT / 32) {
    const int m0 = (u >> 1) * 16, vb0 = (u & 1) * HB;
    if (m0 >= dim || vb0 * 8 >= vdim) continue;
    float acc[HB][4];
#pragma unroll
    for (int i = 0; i < HB; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll 2
    for (int kb = 0; kb < LC / 16; ++kb) {
      // A = K'^T: element (state row m, token k) lies at [k][m]
      uint32_t ah[4], al[4];
      const int tok = kb * 16 + (lane >> 4) * 8 + (lane & 7), dm = m0 + ((lane >> 3) & 1) * 8;
      ldmatrix_x4_trans(ah[0], ah[1], ah[2], ah[3], smem_u32(&Kh[tok][dm]));
      ldmatrix_x4_trans(al[0], al[1], al[2], al[3], smem_u32(&Kl[tok][dm]));
#pragma unroll
      for (int vb = 0; vb < HB; ++vb) {
        uint32_t b0, b1;
        ldmatrix_x2_trans_la(b0, b1, smem_u32(&Vs[kb * 16 + (lane & 15)][(vb0 + vb) * 8]));
        mma_bf16_16816(acc[vb], ah, b0, b1);
        mma_bf16_16816(acc[vb], al, b0, b1);
      }
    }
    const int r = m0 + (lane >> 2), c = (lane & 3) * 2;
#pragma unroll
    for (int vb = 0; vb < HB; ++vb)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int rr = r + (e >> 1) * 8, cc = (vb0 + vb) * 8 + c;
        if (rr >= dim || cc >= vdim) continue;
        float* d = U + (size_t)rr * a.vdim + cc;
        if (a.vdim % 2 == 0) {
          *reinterpret_cast<float2*>(d) = make_float2(acc[vb][e], acc[vb][e + 1]);
        } else {
          d[0] = acc[vb][e];
          if (cc + 1 < vdim) d[1] = acc[vb][e + 1];
        }
      }
  }
}

// CTA (chunk, head): U [dim, vdim] = sum_s decay^(L-1-s) k_scale k_s v_s^T -> ws
template <int DP, int VP>
__global__ void __launch_bounds__(LT) linear_chunk_state_kernel(const LinearAttnArgs a) {
  extern __shared__ __align__(16) unsigned char lc_smem[];
  typedef bf16 KT[DP + 8];
  typedef bf16 VT[VP + 8];
  KT* Kh = reinterpret_cast<KT*>(lc_smem);
  KT* Kl = Kh + LC;
  VT* Vs = reinterpret_cast<VT*>(Kl + LC);
  pdl_wait();
  pdl_trigger();
  int row0, L;
  if (!find_chunk(a, blockIdx.x, &row0, &L)) return;
  const int h = blockIdx.y, dim = a.dim, vdim = a.vdim;
  const float* pw = a.decay_pow + h * (LC + 1);
  {
    TileRegs<DP> k;
    TileRegs<VP> v;
    k.load(a.k_bf + h * dim, a.ld_bf, row0, L, dim);
    v.load(a.v_bf + h * vdim, a.ld_bf, row0, L, vdim);
    v.store(Vs, a.act);
    // decayed keys as hi + lo pairs
#pragma unroll
    for (int n = 0; n < TileRegs<DP>::N; ++n) {
      const int i = threadIdx.x + n * LT, r = i / (DP / 8), c = (i % (DP / 8)) * 8;
      const float f = r < L ? a.k_scale * pw[L - 1 - r] : 0.f;
      const uint32_t u[4] = {k.v[n].x, k.v[n].y, k.v[n].z, k.v[n].w};
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float x0 = lo2f(u[j]), x1 = hi2f(u[j]);
        if (a.act) {  // the activated key is a bf16 value, as in the scores
          const uint32_t act = pack2f(silu_f(x0), silu_f(x1));
          x0 = lo2f(act), x1 = hi2f(act);
        }
        x0 *= f, x1 *= f;
        hi[j] = pack2f(x0, x1);
        lo[j] = pack2f(x0 - lo2f(hi[j]), x1 - hi2f(hi[j]));
      }
      *reinterpret_cast<uint4*>(&Kh[r][c]) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(&Kl[r][c]) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
  }
  __syncthreads();
  chunk_state_product<DP, VP>(a, Kh, Kl, Vs, h, 0);
}

// thread = state element of (segment, head): walks the segment's chunks; the chunk's U becomes its entry state
template <bool GATED>
__global__ void __launch_bounds__(256) linear_carry_kernel(const LinearAttnArgs a) {
  pdl_wait();
  pdl_trigger();
  const int seg = blockIdx.y, per = a.dim * a.vdim, i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= a.heads * per) return;
  int first = 0;
  for (int s = 0; s < seg; ++s) first += (a.seg_start[s + 1] - a.seg_start[s] + LC - 1) / LC;
  const int len = a.seg_start[seg + 1] - a.seg_start[seg], nc = (len + LC - 1) / LC, h = i / per;
  float full = 0.f, last = 0.f;
  if (!GATED) full = a.decay_pow[h * (LC + 1) + LC], last = a.decay_pow[h * (LC + 1) + len - (nc - 1) * LC];
  // gated: the whole decay of a chunk stands in its last row
  const int pitch = gated_decay_pitch(a.dim);
  const size_t crow = (size_t)a.heads * pitch;
  const float* cum = GATED ? a.gate.cum + (size_t)a.seg_start[seg] * crow + (size_t)h * pitch + (i - h * per) / a.vdim : nullptr;
  float* st = a.state + (size_t)a.seg_slot[seg] * a.slot_stride + i;
  const size_t stride = (size_t)a.heads * per;
  float* w = a.ws + (size_t)first * stride + i;
  float S = *st;
  constexpr int PF = 8;  // chunks whose loads are in flight
  float u[PF], f[PF];
  for (int c0 = 0; c0 < nc; c0 += PF) {
#pragma unroll
    for (int j = 0; j < PF; ++j) u[j] = c0 + j < nc ? w[(size_t)(c0 + j) * stride] : 0.f;
    if constexpr (GATED) {
#pragma unroll
      for (int j = 0; j < PF; ++j) f[j] = c0 + j < nc ? cum[(size_t)(min((c0 + j + 1) * LC, len) - 1) * crow] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < PF; ++j) {
      if (c0 + j >= nc) break;
      w[(size_t)(c0 + j) * stride] = S;
      S = fmaf(GATED ? exp2f(f[j]) : c0 + j == nc - 1 ? last : full, S, u[j]);
    }
  }
  *st = S;
}

// the chunk's entry state of head h, value columns v0 .. -> hi and lo tiles [DP][VP + 8], zeros beyond
template <int DP, int VP>
__device__ __forceinline__ void load_entry_state(const LinearAttnArgs& a, int h, int v0, bf16 (*Sh)[VP + 8], bf16 (*Sl)[VP + 8]) {
  const int tid = threadIdx.x, dim = a.dim, vcols = min(VP, a.vdim - v0);
  const float* S = a.ws + ((size_t)blockIdx.x * a.heads + h) * dim * a.vdim + v0;
  if (a.vdim % 4 == 0) {
    constexpr int NS = DP * (VP / 4) / LT, B = 8;
#pragma unroll
    for (int n0 = 0; n0 < NS; n0 += B) {  // (NS is 4, 8 or 16)
      float4 x[B];
#pragma unroll
      for (int j = 0; j < B; ++j) {
        const int i = tid + (n0 + j) * LT, d = i / (VP / 4), c = (i % (VP / 4)) * 4;
        x[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (n0 + j < NS && d < dim && c < vcols) x[j] = *reinterpret_cast<const float4*>(S + (size_t)d * a.vdim + c);
      }
#pragma unroll
      for (int j = 0; j < B; ++j) {
        if (n0 + j >= NS) break;
        const int i = tid + (n0 + j) * LT, d = i / (VP / 4), c = (i % (VP / 4)) * 4;
        const uint32_t h0 = pack2f(x[j].x, x[j].y), h1 = pack2f(x[j].z, x[j].w);
        *reinterpret_cast<uint2*>(&Sh[d][c]) = make_uint2(h0, h1);
        *reinterpret_cast<uint2*>(&Sl[d][c]) =
            make_uint2(pack2f(x[j].x - lo2f(h0), x[j].y - hi2f(h0)), pack2f(x[j].z - lo2f(h1), x[j].w - hi2f(h1)));
      }
    }
  } else {
    for (int i = tid; i < DP * VP; i += LT) {
      const int d = i / VP, c = i % VP;
      const float x = d < dim && c < vcols ? S[(size_t)d * a.vdim + c] : 0.f;
      const bf16 hi = f2bf(x);
      Sh[d][c] = hi, Sl[d][c] = f2bf(x - bf2f(hi));
    }
  }
}

// rows of a chunk, turned around in shared memory -> fp32 rows, or normed per head, weighted, gated bf16 rows; four threads per row write
// whole pieces.  v0: the CTA's first value column
template <int VP>
__device__ __forceinline__ void chunk_epilogue(const LinearAttnArgs& a, const float (*os)[VP + 4], int row0, int L, int h, int v0) {
  const int tid = threadIdx.x, t = tid >> 2, c0 = (tid & 3) * 4, vdim = min(VP, a.vdim - v0);  // value columns of this CTA
  const size_t r = (size_t)(row0 + t);
  float n = 1.f;
  if (a.norm_gate) {
    float q = 0.f;
    for (int c = c0; c < vdim; c += 16)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < vdim) q = fmaf(os[t][c + e], os[t][c + e], q);
    q += __shfl_xor_sync(0xffffffffu, q, 1);
    q += __shfl_xor_sync(0xffffffffu, q, 2);
    n = 1.0f / sqrtf(q / (float)vdim + a.eps);
  }
  if (t >= L) return;
  if (a.norm_gate) {
    const bf16* g = a.g_bf + r * a.ld_bf + h * a.vdim;
    bf16* out = a.out_bf + r * a.ldo_bf + h * a.vdim;
    const bool vec = a.vdim % 4 == 0 && a.ld_bf % 4 == 0 && a.ldo_bf % 4 == 0 && ((reinterpret_cast<uintptr_t>(a.g_bf) | reinterpret_cast<uintptr_t>(a.out_bf)) & 7) == 0;
#pragma unroll 2
    for (int c = c0; c < vdim; c += 16) {
      if (vec) {
        const uint2 gv = *reinterpret_cast<const uint2*>(g + c);
        float4 x = *reinterpret_cast<const float4*>(&os[t][c]);
        if (a.norm_w) x.x *= bf2f(a.norm_w[c]), x.y *= bf2f(a.norm_w[c + 1]), x.z *= bf2f(a.norm_w[c + 2]), x.w *= bf2f(a.norm_w[c + 3]);
        *reinterpret_cast<uint2*>(out + c) = make_uint2(pack2f(x.x * n * silu_f(lo2f(gv.x)), x.y * n * silu_f(hi2f(gv.x))),
                                                        pack2f(x.z * n * silu_f(lo2f(gv.y)), x.w * n * silu_f(hi2f(gv.y))));
      } else {
        for (int e = c; e < min(c + 4, vdim); ++e) out[e] = f2bf(os[t][e] * n * (a.norm_w ? bf2f(a.norm_w[e]) : 1.f) * silu_f(bf2f(g[e])));
      }
    }
  } else {
    float* out = a.out + r * a.ldo + h * a.vdim + v0;
    const bool vec = a.vdim % 4 == 0 && a.ldo % 4 == 0 && (reinterpret_cast<uintptr_t>(a.out) & 15) == 0;
#pragma unroll 2
    for (int c = c0; c < vdim; c += 16) {
      if (vec) *reinterpret_cast<float4*>(out + c) = *reinterpret_cast<const float4*>(&os[t][c]);
      else
        for (int e = c; e < min(c + 4, vdim); ++e) out[e] = os[t][e];
    }
  }
}

// CTA (chunk, head): the outputs of the chunk's rows from its entry state and its own keys and values; warp w owns rows
// 16 (w % 4) .. and half w / 4 of the value columns
template <int DP, int VP>
__global__ void __launch_bounds__(LT) linear_chunk_out_kernel(const LinearAttnArgs a) {
  extern __shared__ __align__(16) unsigned char lc_smem[];
  typedef bf16 KT[DP + 8];
  typedef bf16 VT[VP + 8];
  KT* Qs = reinterpret_cast<KT*>(lc_smem);
  KT* Ks = Qs + LC;
  VT* Vs = reinterpret_cast<VT*>(Ks + LC);
  VT* Sh = Vs + LC;   // [DP] entry state, hi
  VT* Sl = Sh + DP;   // lo
  __shared__ float pw[LC + 1];
  pdl_wait();
  pdl_trigger();
  int row0, L;
  if (!find_chunk(a, blockIdx.x, &row0, &L)) return;
  const int h = blockIdx.y, dim = a.dim, vdim = a.vdim, tid = threadIdx.x;
  {
    TileRegs<DP> q, k;
    TileRegs<VP> v;
    q.load(a.q_bf + h * dim, a.ld_bf, row0, L, dim);
    k.load(a.k_bf + h * dim, a.ld_bf, row0, L, dim);
    v.load(a.v_bf + h * vdim, a.ld_bf, row0, L, vdim);
    for (int i = tid; i <= LC; i += LT) pw[i] = a.decay_pow[h * (LC + 1) + i];
    q.store(Qs, a.act);
    k.store(Ks, a.act);
    v.store(Vs, a.act);
  }
  load_entry_state<DP, VP>(a, h, 0, Sh, Sl);
  __syncthreads();
  constexpr int HB = VP / 16;  // blocks of 8 columns per half
  const int warp = tid >> 5, lane = tid & 31, w0 = (warp & 3) * 16, vb0 = (warp >> 2) * HB;
  const bool active = w0 < L;
  const int qr = lane >> 2, qc = (lane & 3) * 2;
  const int t0 = w0 + qr, t1 = t0 + 8;  // this thread's two rows of the chunk
  float o[HB][4];
#pragma unroll
  for (int i = 0; i < HB; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  if (active) {
    float s[LC / 8][4];
#pragma unroll
    for (int i = 0; i < LC / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll 2
    for (int kk = 0; kk < DP / 16; ++kk) {
      uint32_t qf[4];
      ldmatrix_x4(qf[0], qf[1], qf[2], qf[3], smem_u32(&Qs[w0 + (lane & 15)][kk * 16 + (lane >> 4) * 8]));
#pragma unroll
      for (int nb = 0; nb < LC / 8; ++nb) {
        if (nb * 8 > w0 + 15) break;  // later than every row of the warp
        uint32_t b0, b1;
        ldmatrix_x2(b0, b1, smem_u32(&Ks[nb * 8 + (lane & 7)][kk * 16 + ((lane >> 3) & 1) * 8]));
        mma_bf16_16816(s[nb], qf, b0, b1);
      }
#pragma unroll
      for (int vb = 0; vb < HB; ++vb) {
        uint32_t b0, b1;
        ldmatrix_x2_trans_la(b0, b1, smem_u32(&Sh[kk * 16 + (lane & 15)][(vb0 + vb) * 8]));
        mma_bf16_16816(o[vb], qf, b0, b1);
        ldmatrix_x2_trans_la(b0, b1, smem_u32(&Sl[kk * 16 + (lane & 15)][(vb0 + vb) * 8]));
        mma_bf16_16816(o[vb], qf, b0, b1);
      }
    }
    {
      const float e0 = pw[t0 + 1], e1 = pw[t1 + 1];
#pragma unroll
      for (int vb = 0; vb < HB; ++vb) o[vb][0] *= e0, o[vb][1] *= e0, o[vb][2] *= e1, o[vb][3] *= e1;
    }
#pragma unroll
    for (int kb = 0; kb < LC / 16; ++kb) {
      if (kb * 16 > w0 + 15) break;
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int nb = 2 * kb + (f >> 1), j = nb * 8 + qc, t = (f & 1) ? t1 : t0;
        const float x0 = j <= t ? s[nb][(f & 1) * 2] * (a.k_scale * pw[t - j]) : 0.f;
        const float x1 = j + 1 <= t ? s[nb][(f & 1) * 2 + 1] * (a.k_scale * pw[t - j - 1]) : 0.f;
        ph[f] = pack2f(x0, x1);
        pl[f] = pack2f(x0 - lo2f(ph[f]), x1 - hi2f(ph[f]));
      }
#pragma unroll
      for (int vb = 0; vb < HB; ++vb) {
        uint32_t b0, b1;
        ldmatrix_x2_trans_la(b0, b1, smem_u32(&Vs[kb * 16 + (lane & 15)][(vb0 + vb) * 8]));
        mma_bf16_16816(o[vb], ph, b0, b1);
        mma_bf16_16816(o[vb], pl, b0, b1);
      }
    }
  }
  // the result goes through shared memory (everything else there has been read): four threads per row then write whole pieces
  float (*os)[VP + 4] = reinterpret_cast<float (*)[VP + 4]>(lc_smem);
  __syncthreads();
  if (active) {
#pragma unroll
    for (int vb = 0; vb < HB; ++vb) {
      const int c = (vb0 + vb) * 8 + qc;
      *reinterpret_cast<float2*>(&os[t0][c]) = make_float2(o[vb][0], o[vb][1]);
      *reinterpret_cast<float2*>(&os[t1][c]) = make_float2(o[vb][2], o[vb][3]);
    }
  }
  __syncthreads();
  chunk_epilogue<VP>(a, os, row0, L, h, 0);
}

// ---------------------------------------------------------------- gated channels
__device__ __forceinline__ float ex2(float x) {  // 2^x, results below the normal range become 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// CTA (chunk, 64 channels): log2 of the decays of the chunk's rows, summed up row by row -> cum [n, heads, pitch].  A thread walks a block of
// 16 rows of one channel, the blocks' sums meet in shared memory; RMAX: the low-rank map's row in registers (0: any rank, from memory)
constexpr int GD_CH = 64, GD_ROWS = 16, GD_PARTS = LC / GD_ROWS;
template <int RMAX>
__global__ void __launch_bounds__(GD_CH * GD_PARTS) gated_decay_kernel(const LinearAttnArgs a) {
  extern __shared__ __align__(16) float gd_low[];  // [LC][RP] low-rank rows, zeros beyond the rank
  __shared__ float sums[GD_PARTS][GD_CH];
  pdl_wait();
  pdl_trigger();
  int row0, L;
  if (!find_chunk(a, blockIdx.x, &row0, &L)) return;
  const GatedDecay& g = a.gate;
  const int rank = g.rank, RP = RMAX > 0 ? RMAX : rank, pitch = gated_decay_pitch(a.dim);
  for (int i = threadIdx.x; i < L * RP; i += GD_CH * GD_PARTS) {
    const int t = i / RP, j = i - t * RP;
    gd_low[i] = j >= rank ? 0.f : g.low_bf ? bf2f(g.low_bf[(size_t)(row0 + t) * a.ld_bf + j]) : g.low[(size_t)(row0 + t) * a.ld + j];
  }
  const int c = threadIdx.x % GD_CH, part = threadIdx.x / GD_CH, at = blockIdx.y * GD_CH + c, h = at / pitch, d = at - h * pitch;
  const bool live = h < a.heads && d < a.dim;
  const int ch = live ? h * a.dim + d : 0;
  float w[RMAX > 0 ? RMAX : 1];
  if constexpr (RMAX > 0) {
#pragma unroll
    for (int j = 0; j < RMAX; ++j) w[j] = j < rank ? bf2f(g.a2[(size_t)ch * rank + j]) : 0.f;
  }
  const float bias = bf2f(g.bias[ch]);
  __syncthreads();
  float b[GD_ROWS], sum = 0.f;  // running sums of the thread's rows
#pragma unroll
  for (int k = 0; k < GD_ROWS; ++k) {
    const int t = part * GD_ROWS + k;
    float z = bias;
    if (t < L) {
      const float* low = gd_low + t * RP;
      if constexpr (RMAX > 0) {
#pragma unroll
        for (int j = 0; j < RMAX; j += 4) {
          const float4 x = *reinterpret_cast<const float4*>(low + j);
          z = fmaf(w[j], x.x, z), z = fmaf(w[j + 1], x.y, z), z = fmaf(w[j + 2], x.z, z), z = fmaf(w[j + 3], x.w, z);
        }
      } else {
        for (int j = 0; j < rank; ++j) z = fmaf(bf2f(g.a2[(size_t)ch * rank + j]), low[j], z);
      }
      if (live) sum += log2_sigmoid_pow(z, g.inv_tau);
    }
    b[k] = sum;
  }
  sums[part][c] = sum;
  __syncthreads();
  float before = 0.f;
  for (int p = 0; p < part; ++p) before += sums[p][c];
  if (h >= a.heads) return;
  float* out = g.cum + (size_t)row0 * a.heads * pitch + at;
#pragma unroll
  for (int k = 0; k < GD_ROWS; ++k) {
    const int t = part * GD_ROWS + k;
    if (t < L) out[(size_t)t * a.heads * pitch] = before + b[k];
  }
}

// eight running sums of one row from channel c on (pitch is a multiple of 4; zeros beyond it)
__device__ __forceinline__ void load_cum8(const float* row, int c, int pitch, float (&b)[8]) {
  float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
  if (c < pitch) x = *reinterpret_cast<const float4*>(row + c);
  if (c + 4 < pitch) y = *reinterpret_cast<const float4*>(row + c + 4);
  b[0] = x.x, b[1] = x.y, b[2] = x.z, b[3] = x.w, b[4] = y.x, b[5] = y.y, b[6] = y.z, b[7] = y.w;
}

// CTA (chunk, head, VP value columns): U [dim, vdim] = sum_s (k_s 2^(b_last - b_s)) v_s^T -> ws
template <int DP, int VP>
__global__ void __launch_bounds__(LT) gated_chunk_state_kernel(const LinearAttnArgs a) {
  extern __shared__ __align__(16) unsigned char lc_smem[];
  typedef bf16 KT[DP + 8];
  typedef bf16 VT[VP + 8];
  KT* Kh = reinterpret_cast<KT*>(lc_smem);
  KT* Kl = Kh + LC;
  VT* Vs = reinterpret_cast<VT*>(Kl + LC);
  pdl_wait();
  pdl_trigger();
  int row0, L;
  if (!find_chunk(a, blockIdx.x, &row0, &L)) return;
  const int h = blockIdx.y, v0 = blockIdx.z * VP, dim = a.dim, pitch = gated_decay_pitch(dim);
  {
    TileRegs<DP> k;
    TileRegs<VP> v;
    k.load(a.k_bf + h * dim, a.ld_bf, row0, L, dim);
    v.load(a.v_bf + h * a.vdim + v0, a.ld_bf, row0, L, min(VP, a.vdim - v0));
    const size_t crow = (size_t)a.heads * pitch;
    const float* cum = a.gate.cum + (size_t)row0 * crow + (size_t)h * pitch;
    float b[TileRegs<DP>::N][8], bl[8];
#pragma unroll
    for (int n = 0; n < TileRegs<DP>::N; ++n) {
      const int i = threadIdx.x + n * LT, r = i / (DP / 8), c = (i % (DP / 8)) * 8;
      load_cum8(cum + (size_t)min(r, L - 1) * crow, c, pitch, b[n]);
      if (n == 0) load_cum8(cum + (size_t)(L - 1) * crow, c, pitch, bl);  // LT is a multiple of DP / 8: the same columns in every round
    }
    v.store(Vs, a.act);
#pragma unroll
    for (int n = 0; n < TileRegs<DP>::N; ++n) {
      const int i = threadIdx.x + n * LT, r = i / (DP / 8), c = (i % (DP / 8)) * 8;
      const uint32_t u[4] = {k.v[n].x, k.v[n].y, k.v[n].z, k.v[n].w};
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float x0 = lo2f(u[j]), x1 = hi2f(u[j]);
        if (a.act) {  // the activated key is a bf16 value, as in the scores
          const uint32_t act = pack2f(silu_f(x0), silu_f(x1));
          x0 = lo2f(act), x1 = hi2f(act);
        }
        x0 *= a.k_scale * ex2(bl[2 * j] - b[n][2 * j]), x1 *= a.k_scale * ex2(bl[2 * j + 1] - b[n][2 * j + 1]);
        hi[j] = pack2f(x0, x1);
        lo[j] = pack2f(x0 - lo2f(hi[j]), x1 - hi2f(hi[j]));
      }
      *reinterpret_cast<uint4*>(&Kh[r][c]) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(&Kl[r][c]) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
  }
  __syncthreads();
  chunk_state_product<DP, VP>(a, Kh, Kl, Vs, h, v0);
}

// CTA (chunk, head, VP value columns): the outputs of the chunk's rows.  Warp w owns the block of rows 16 (w % 4) .. and half w / 4 of the
// value columns; decayed queries and keys are made in registers, from the bf16 rows and the running sums in shared memory.
constexpr float GATED_RANGE = 100.f;  // largest range of log2 decays inside a block of 16 rows that the factored form takes
template <int DP, int VP>
__global__ void __launch_bounds__(LT) gated_chunk_out_kernel(const LinearAttnArgs a) {
  extern __shared__ __align__(16) unsigned char lc_smem[];
  typedef bf16 KT[DP + 8];
  typedef bf16 VT[VP + 8];
  typedef float BT[DP + 4];
  KT* Qs = reinterpret_cast<KT*>(lc_smem);
  KT* Ks = Qs + LC;
  VT* Vs = reinterpret_cast<VT*>(Ks + LC);
  VT* Sh = Vs + LC;  // [DP] entry state, hi
  VT* Sl = Sh + DP;  // lo
  BT* Bs = reinterpret_cast<BT*>(Sl + DP);  // running sums
  __shared__ float tab[3][LC / 16][DP];     // per block of 16 rows: 2^b of its first row | 2^(half its range) | the middle of its range
  __shared__ int wide[LC / 16];             // the block's range is too long for the factored form
  pdl_wait();
  pdl_trigger();
  int row0, L;
  if (!find_chunk(a, blockIdx.x, &row0, &L)) return;
  const int h = blockIdx.y, v0 = blockIdx.z * VP, dim = a.dim, tid = threadIdx.x, pitch = gated_decay_pitch(dim);
  if (tid < LC / 16) wide[tid] = 0;
  {
    TileRegs<DP> q, k;
    TileRegs<VP> v;
    q.load(a.q_bf + h * dim, a.ld_bf, row0, L, dim);
    k.load(a.k_bf + h * dim, a.ld_bf, row0, L, dim);
    v.load(a.v_bf + h * a.vdim + v0, a.ld_bf, row0, L, min(VP, a.vdim - v0));
    const size_t crow = (size_t)a.heads * pitch;
    const float* cum = a.gate.cum + (size_t)row0 * crow + (size_t)h * pitch;
    constexpr int NB = LC * (DP / 4) / LT;
    float4 b[NB];
#pragma unroll
    for (int n = 0; n < NB; ++n) {
      const int i = tid + n * LT, r = i / (DP / 4), c = (i % (DP / 4)) * 4;
      b[n] = c < pitch ? *reinterpret_cast<const float4*>(cum + (size_t)min(r, L - 1) * crow + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    load_entry_state<DP, VP>(a, h, v0, Sh, Sl);  // on its way together with the tiles
    q.store(Qs, a.act);
    k.store(Ks, a.act);
    v.store(Vs, a.act);
#pragma unroll
    for (int n = 0; n < NB; ++n) {
      const int i = tid + n * LT;
      *reinterpret_cast<float4*>(&Bs[i / (DP / 4)][(i % (DP / 4)) * 4]) = b[n];
    }
  }
  __syncthreads();
  for (int i = tid; i < LC / 16 * DP; i += LT) {
    const int blk = i / DP, c = i - blk * DP;
    const float first = Bs[blk * 16][c], last = Bs[blk * 16 + 15][c], range = first - last;
    tab[0][blk][c] = ex2(first);
    tab[1][blk][c] = ex2(fminf(0.5f * range, GATED_RANGE));
    tab[2][blk][c] = 0.5f * (first + last);
    if (range > GATED_RANGE) wide[blk] = 1;
  }
  __syncthreads();
  constexpr int HB = VP / 16;  // blocks of 8 columns per half
  const int warp = tid >> 5, lane = tid & 31, blk = warp & 3, w0 = blk * 16, vb0 = (warp >> 2) * HB;
  const bool active = w0 < L, factored = !wide[blk];
  const int qr = lane >> 2, qc = (lane & 3) * 2;
  const int t0 = w0 + qr, t1 = t0 + 8;  // this thread's two rows of the chunk
  float o[HB][4];
#pragma unroll
  for (int i = 0; i < HB; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  if (active) {
    float s[LC / 8][4];
#pragma unroll
    for (int i = 0; i < LC / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    // x [4][2]: an A operand (registers, element pairs) -> hi + lo
    auto split = [](const float (&x)[4][2], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        hi[f] = pack2f(x[f][0], x[f][1]);
        lo[f] = pack2f(x[f][0] - lo2f(hi[f]), x[f][1] - hi2f(hi[f]));
      }
    };
#pragma unroll 1
    for (int kk = 0; kk < DP / 16; ++kk) {
      const int c = kk * 16 + qc;
      // queries decayed from the block's first row on: element pair f is row t0 (f even) or t1, channels c (f < 2) or c + 8
      float x[4][2];
      float2 ref[2];
#pragma unroll
      for (int g = 0; g < 2; ++g) ref[g] = *reinterpret_cast<const float2*>(&Bs[w0][c + 8 * g]);
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int t = (f & 1) ? t1 : t0, cc = c + (f >> 1) * 8;
        const uint32_t u = *reinterpret_cast<const uint32_t*>(&Qs[t][cc]);
        const float2 b = *reinterpret_cast<const float2*>(&Bs[t][cc]);
        x[f][0] = lo2f(u) * a.q_scale * ex2(b.x - ref[f >> 1].x), x[f][1] = hi2f(u) * a.q_scale * ex2(b.y - ref[f >> 1].y);
      }
      uint32_t ah[4], al[4];
      {  // against the entry state
        float y[4][2];
#pragma unroll
        for (int f = 0; f < 4; ++f) {
          const float2 e = *reinterpret_cast<const float2*>(&tab[0][blk][c + (f >> 1) * 8]);
          y[f][0] = x[f][0] * e.x, y[f][1] = x[f][1] * e.y;
        }
        split(y, ah, al);
#pragma unroll
        for (int vb = 0; vb < HB; ++vb) {
          uint32_t b0, b1;
          ldmatrix_x2_trans_la(b0, b1, smem_u32(&Sh[kk * 16 + (lane & 15)][(vb0 + vb) * 8]));
          mma_bf16_16816(o[vb], ah, b0, b1);
          mma_bf16_16816(o[vb], al, b0, b1);
          ldmatrix_x2_trans_la(b0, b1, smem_u32(&Sl[kk * 16 + (lane & 15)][(vb0 + vb) * 8]));
          mma_bf16_16816(o[vb], ah, b0, b1);
        }
      }
      // eight keys from key j0 on, decayed by 2^(r - b), against the queries in ah / al
      auto against = [&](float (&acc)[4], int j0, const float2 (&r)[2]) {
        const int j = j0 + qr;
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          const uint32_t u = *reinterpret_cast<const uint32_t*>(&Ks[j][c + 8 * g]);
          const float2 b = *reinterpret_cast<const float2*>(&Bs[j][c + 8 * g]);
          const float y0 = lo2f(u) * ex2(r[g].x - b.x), y1 = hi2f(u) * ex2(r[g].y - b.y);
          bh[g] = pack2f(y0, y1);
          bl[g] = pack2f(y0 - lo2f(bh[g]), y1 - hi2f(bh[g]));
        }
        mma_bf16_16816(acc, ah, bh[0], bh[1]);
        mma_bf16_16816(acc, al, bh[0], bh[1]);
        mma_bf16_16816(acc, ah, bl[0], bl[1]);
      };
      split(x, ah, al);
#pragma unroll
      for (int nb = 0; nb < LC / 8 - 2; ++nb) {  // keys of earlier blocks
        if (nb * 8 >= w0) break;
        against(s[nb], nb * 8, ref);
      }
      if (factored) {  // keys of the block itself, around the middle of its range
        float2 mid[2];
#pragma unroll
        for (int g = 0; g < 2; ++g) mid[g] = *reinterpret_cast<const float2*>(&tab[2][blk][c + 8 * g]);
#pragma unroll
        for (int f = 0; f < 4; ++f) {
          const float2 e = *reinterpret_cast<const float2*>(&tab[1][blk][c + (f >> 1) * 8]);
          x[f][0] *= e.x, x[f][1] *= e.y;
        }
        split(x, ah, al);
#pragma unroll
        for (int nb = 0; nb < LC / 8; ++nb)
          if ((nb >> 1) == blk) against(s[nb], nb * 8, mid);
      }
    }
    if (!factored) {
#pragma unroll
      for (int nb = 0; nb < LC / 8; ++nb) {
        if ((nb >> 1) != blk) continue;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = (e >> 1) ? t1 : t0, j = nb * 8 + qc + (e & 1);
          float v = 0.f;
          if (j <= t)
#pragma unroll 1
            for (int d = 0; d < dim; ++d) v = fmaf(bf2f(Qs[t][d]) * bf2f(Ks[j][d]), ex2(Bs[t][d] - Bs[j][d]), v);
          s[nb][e] = v * a.q_scale;
        }
      }
    }
#pragma unroll
    for (int kb = 0; kb < LC / 16; ++kb) {
      if (kb > blk) break;
      float x[4][2];
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int nb = 2 * kb + (f >> 1), j = nb * 8 + qc, t = (f & 1) ? t1 : t0;
        x[f][0] = j <= t ? s[nb][(f & 1) * 2] * a.k_scale : 0.f, x[f][1] = j + 1 <= t ? s[nb][(f & 1) * 2 + 1] * a.k_scale : 0.f;
      }
      split(x, ph, pl);
#pragma unroll
      for (int vb = 0; vb < HB; ++vb) {
        uint32_t b0, b1;
        ldmatrix_x2_trans_la(b0, b1, smem_u32(&Vs[kb * 16 + (lane & 15)][(vb0 + vb) * 8]));
        mma_bf16_16816(o[vb], ph, b0, b1);
        mma_bf16_16816(o[vb], pl, b0, b1);
      }
    }
  }
  // the result goes through shared memory (everything else there has been read)
  float (*os)[VP + 4] = reinterpret_cast<float (*)[VP + 4]>(lc_smem);
  __syncthreads();
  if (active) {
#pragma unroll
    for (int vb = 0; vb < HB; ++vb) {
      const int c = (vb0 + vb) * 8 + qc;
      *reinterpret_cast<float2*>(&os[t0][c]) = make_float2(o[vb][0], o[vb][1]);
      *reinterpret_cast<float2*>(&os[t1][c]) = make_float2(o[vb][2], o[vb][3]);
    }
  }
  __syncthreads();
  chunk_epilogue<VP>(a, os, row0, L, h, v0);
}

template <int DP, int VP>
cudaError_t launch_gated_chunked(const LinearAttnArgs& a, cudaStream_t st) {
  const int chunks = a.n_rows / LC + a.n_seg, nvb = (a.vdim + VP - 1) / VP;  // chunks: an upper bound
  const size_t s1 = ((size_t)2 * LC * (DP + 8) + (size_t)LC * (VP + 8)) * sizeof(bf16);
  const size_t s2 = ((size_t)2 * LC * (DP + 8) + (size_t)(LC + 2 * DP) * (VP + 8)) * sizeof(bf16) + (size_t)LC * (DP + 4) * sizeof(float);
  static PerDeviceOnce once;
  cudaError_t r;
  if (once.need()) {
    if ((r = cudaFuncSetAttribute(gated_chunk_state_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1)) != cudaSuccess) return r;
    if ((r = cudaFuncSetAttribute(gated_chunk_out_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2)) != cudaSuccess) return r;
    once.done();
  }
  const int rank = a.gate.rank, RP = rank <= 16 ? 16 : rank <= 32 ? 32 : rank;
  const dim3 dgrid(chunks, (a.heads * gated_decay_pitch(a.dim) + GD_CH - 1) / GD_CH);
  auto* decay = rank <= 16 ? gated_decay_kernel<16> : rank <= 32 ? gated_decay_kernel<32> : gated_decay_kernel<0>;
  if ((r = launch_k(decay, dgrid, dim3(GD_CH * GD_PARTS), (size_t)LC * RP * sizeof(float), st, a)) != cudaSuccess) return r;
  if ((r = launch_k(gated_chunk_state_kernel<DP, VP>, dim3(chunks, a.heads, nvb), dim3(LT), s1, st, a)) != cudaSuccess) return r;
  const int per = a.heads * a.dim * a.vdim;
  if ((r = launch_k(linear_carry_kernel<true>, dim3((per + 255) / 256, a.n_seg), dim3(256), 0, st, a)) != cudaSuccess) return r;
  return launch_k(gated_chunk_out_kernel<DP, VP>, dim3(chunks, a.heads, nvb), dim3(LT), s2, st, a);
}

template <int DP, int VP>
cudaError_t launch_chunked(const LinearAttnArgs& a, cudaStream_t st) {
  const int chunks = a.n_rows / LC + a.n_seg;  // upper bound
  const size_t s1 = ((size_t)2 * LC * (DP + 8) + (size_t)LC * (VP + 8)) * sizeof(bf16);
  const size_t s2 = ((size_t)2 * LC * (DP + 8) + (size_t)(LC + 2 * DP) * (VP + 8)) * sizeof(bf16);
  static PerDeviceOnce once;
  if (once.need()) {
    cudaError_t r;
    if ((r = cudaFuncSetAttribute(linear_chunk_state_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1)) != cudaSuccess) return r;
    if ((r = cudaFuncSetAttribute(linear_chunk_out_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2)) != cudaSuccess) return r;
    once.done();
  }
  cudaError_t r = launch_k(linear_chunk_state_kernel<DP, VP>, dim3(chunks, a.heads), dim3(LT), s1, st, a);
  if (r != cudaSuccess) return r;
  const int per = a.heads * a.dim * a.vdim;
  if ((r = launch_k(linear_carry_kernel<false>, dim3((per + 255) / 256, a.n_seg), dim3(256), 0, st, a)) != cudaSuccess) return r;
  return launch_k(linear_chunk_out_kernel<DP, VP>, dim3(chunks, a.heads), dim3(LT), s2, st, a);
}

}  // namespace

bool linear_attention_chunked(const LinearAttnArgs& a) {
  const bool gated = a.gate.a2 != nullptr;
  return a.q_bf && a.k_bf && a.v_bf && a.n_rows >= LC && a.dim <= 128 && a.ws && linear_ws_floats(a.n_rows, a.n_seg, a.heads, a.dim, a.vdim) <= a.ws_floats &&
         (gated ? a.gate.cum && a.gate.low_bf && a.gate.rank <= 160 : a.vdim <= 128 && a.q_scale == 1.f);
}

bool linear_attention_norm_fits(const LinearAttnArgs& a) { return linear_attention_chunked(a) && a.vdim <= 128; }

cudaError_t launch_linear_attention(const LinearAttnArgs& a, cudaStream_t st, int* n_launches) {
  if (n_launches) *n_launches = 0;
  if (a.n_rows <= 0 || a.n_seg <= 0) return cudaSuccess;
  const bool gated = a.gate.a2 != nullptr;
  if (a.heads <= 0 || a.dim <= 0 || a.vdim <= 0 || !a.state || !(a.q_bf || a.q)) return cudaErrorInvalidValue;
  if (gated ? (a.gate.rank <= 0 || !a.gate.bias || !(a.q_bf ? a.gate.low_bf != nullptr : a.gate.low != nullptr)) : !a.decay_pow) return cudaErrorInvalidValue;
  const bool chunked = linear_attention_chunked(a);
  if (a.norm_gate ? (!linear_attention_norm_fits(a) || !a.g_bf || !a.out_bf) : !a.out) return cudaErrorInvalidValue;
  if (chunked && gated) {
    if (n_launches) *n_launches = 4;
    if (a.dim <= 64) return a.vdim <= 64 ? launch_gated_chunked<64, 64>(a, st) : launch_gated_chunked<64, 128>(a, st);
    return a.vdim <= 64 ? launch_gated_chunked<128, 64>(a, st) : launch_gated_chunked<128, 128>(a, st);
  }
  if (chunked) {
    if (n_launches) *n_launches = 3;
    if (a.dim <= 64) return a.vdim <= 64 ? launch_chunked<64, 64>(a, st) : launch_chunked<64, 128>(a, st);
    return a.vdim <= 64 ? launch_chunked<128, 64>(a, st) : launch_chunked<128, 128>(a, st);
  }
  const int parts = (a.dim + LA_NR - 1) / LA_NR;
  if (parts > 32) return cudaErrorInvalidValue;  // head sizes up to 256
  if (n_launches) *n_launches = 1;
  const size_t smem = ((size_t)LA_TOK * (gated ? 3 : 2) * parts * LA_NR + LA_TOK * 32 + (size_t)LA_TOK * parts * 32) * sizeof(float);
  auto* kern = gated ? linear_scan_kernel<true> : linear_scan_kernel<false>;
  if (smem > 48 * 1024) {
    cudaError_t r = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
    if (r != cudaSuccess) return r;
  }
  return launch_k(kern, dim3(a.heads, (a.vdim + 31) / 32, a.n_seg), dim3(32 * parts), smem, st, a, parts);
}

}  // namespace qie
