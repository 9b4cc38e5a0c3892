// gebadra.h -- the Gebadra model family: a decoder that carries several copies of the residual stream
// (hyper-connections) behind layer norms with bias, and whose layers mix by one of
//  * lightning attention: linear attention with a fixed decay per head over SiLU-activated queries, keys and values, the
//    concatenated heads RMS-normed together and gated by a sigmoid;
//  * a parallel block: grouped-query softmax attention beside retention, both reading the same input, each output
//    RMS-normed over the width, half of their sum added.  The attention norms its queries and keys over the whole
//    projection, rotates them (neighbouring pairs, linearly scaled positions), sees a sliding window of tokens and one
//    mean key and value per block of tokens before it, and mixes the heads' softmax weights; retention is the linear
//    recurrence without activations, a unit RMS norm per head and a SiLU gate.
// A dense SiLU-gated feed-forward follows (or none).  A layer may use another layer's weights with a cache and state of
// its own.  Streams, norms, scores, softmax weights and their mix, angles, recurrent state and decays are fp32.
//
// The mechanisms are launchers with their constants as arguments: the linear recurrence (linear_attn.cu) and the norm
// behind it (rmsnorm_f32.cu) here; the layer norm and the two normed outputs of a hyper-connection step (hyper.cu), the
// whole-projection norm, pooled rows and mixed softmax weights of the paged attention (attn_gqa.cu) in fosavik.h, the gated
// activation in dedunex.h.  gebadra_model.cu holds the configuration reader, the weight loader and the launch order.  The
// family shares the engine's sequences, page allocator, block tables, row metadata, sampler, scheduler and C ABI with the
// other families.
#pragma once
#include <cuda_runtime.h>

#include <string>
#include <vector>

#include "common.cuh"
#include "dedunex.h"
#include "family.h"
#include "fosavik.h"
#include "nogatar.h"

struct qie_engine;

namespace qie {

// ---------------------------------------------------------------- linear attention with a fixed or a gated decay (linear_attn.cu)
// Per head h over the rows of each segment, state S [dim, vdim] of slot s at state + s * slot_stride + h * dim * vdim (fp32, carried):
//   S = diag(decay) S + (k_scale k_t) v_t^T,   o_t = S^T (q_scale q_t)          with act 1: q, k, v = silu of the rows read
// q [n, heads * dim], k alike, v [n, heads * vdim] are columns of fp32 rows (row stride ld) or of bf16 rows (*_bf, ld_bf).
// The decay is one fixed number per head, or (gate.a2 != null) one per key channel that every token gates:
//   decay_pow: [heads][LINEAR_CHUNK + 1] the powers decay_h^0 .. decay_h^LINEAR_CHUNK on the device
//   gate:      decay_t[h, d] = sigmoid(z)^inv_tau, z = a2[h * dim + d, :] . low_t + bias[h * dim + d], low_t the token's low-rank row
// The result goes to fp32 rows.  With norm_gate (only where linear_attention_norm_fits says so) each head's o is divided by
// sqrt(mean(o^2) + eps), multiplied by norm_w (null: 1) and silu(g_bf[t, h * vdim + c]) and written as bf16 rows instead.
// bf16 sources, LINEAR_CHUNK rows and more and a workspace: portions run in chunks of LINEAR_CHUNK rows on tensor cores (each chunk's own
// contribution to the state, a carry pass over the chunks, then the outputs of all chunks side by side); else token by token.
constexpr int LINEAR_CHUNK = 64;
struct GatedDecay {
  const float* low = nullptr;  // [n, rank] columns of fp32 rows (row stride LinearAttnArgs::ld) or of bf16 rows (low_bf, ld_bf)
  const bf16* low_bf = nullptr;
  int rank = 0;
  const bf16* a2 = nullptr;    // [heads * dim, rank]
  const bf16* bias = nullptr;  // [heads * dim]
  float inv_tau = 1.f;
  float* cum = nullptr;  // workspace of the chunked form, gated_decay_floats(): log2 of the decays, summed up inside every chunk
};
__host__ __device__ inline int gated_decay_pitch(int dim) { return (dim + 3) / 4 * 4; }  // floats per head and row
inline size_t gated_decay_floats(size_t rows, int heads, int dim) { return rows * heads * gated_decay_pitch(dim); }
struct LinearAttnArgs {
  const float *q = nullptr, *k = nullptr, *v = nullptr;
  int ld = 0;
  const bf16 *q_bf = nullptr, *k_bf = nullptr, *v_bf = nullptr;
  int ld_bf = 0;
  int act = 0;
  float k_scale = 1.f, q_scale = 1.f;
  int heads = 0, dim = 0, vdim = 0;
  const float* decay_pow = nullptr;
  GatedDecay gate;
  float* out = nullptr;
  int ldo = 0;
  int norm_gate = 0;
  const bf16* g_bf = nullptr;  // row stride ld_bf
  const bf16* norm_w = nullptr;  // [vdim], the same for every head
  float eps = 0.f;
  bf16* out_bf = nullptr;
  int ldo_bf = 0;
  float* state = nullptr;
  size_t slot_stride = 0;
  const int* seg_start = nullptr;
  const int* seg_slot = nullptr;
  int n_seg = 0, n_rows = 0;
  float* ws = nullptr;  // linear_ws_floats
  size_t ws_floats = 0;
};
inline size_t linear_ws_floats(size_t rows, size_t segs, int heads, int dim, int vdim) {
  return (rows / LINEAR_CHUNK + segs + 1) * heads * (size_t)dim * vdim;
}
// does the chunked form run, and can norm_gate be asked for (one CTA holds a head's values whole)?
bool linear_attention_chunked(const LinearAttnArgs& a);
bool linear_attention_norm_fits(const LinearAttnArgs& a);
cudaError_t launch_linear_attention(const LinearAttnArgs& a, cudaStream_t st, int* n_launches = nullptr);

// ---------------------------------------------------------------- norm, then gate (rmsnorm_f32.cu)
// out[r, c] = v[r, c] / sqrt(mean_group(v[r]^2) + eps) * w[c] * act(g[r, c]);  `groups` equal parts of `width`; w null: 1
// (w_shared: w holds one part's weights, the same for every part);
// act 0: silu, 1: sigmoid.  g: fp32 rows or bf16 rows; the result goes to fp32 rows and / or bf16 rows.
struct NormGate {
  const float* v = nullptr;
  int ldv = 0;
  const float* g = nullptr;
  int ldg = 0;
  const bf16* g_bf = nullptr;
  int ldg_bf = 0;
  const bf16* w = nullptr;
  int width = 0, groups = 1, act = 0, n = 0, w_shared = 0;
  float eps = 0.f;
  float* out = nullptr;
  int ldo = 0;
  bf16* out_bf = nullptr;
  int ldo_bf = 0;
};
cudaError_t launch_norm_gate(const NormGate& a, cudaStream_t st);

// ---------------------------------------------------------------- the model (gebadra_model.cu)
struct GbLinear {  // lightning, or the right half of a parallel layer
  int heads = 0, dim = 0, vdim = 0;
  std::vector<double> decay;
  const float* decay_pow = nullptr;  // device
};
struct GbLayer {
  int type = 0;          // 0 lightning, 1 parallel
  int weights_of = -1;   // >= 0: the layer whose tensors this one uses
  GbLinear lin;
  // parallel: left half
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, window = 0, pool = 0;
  float scale = 1.f;
  RotaryCfg rot;
  int rope_id = -1;
  int ff = 0;  // feed-forward (0 = none)
  // the input projection as one matrix: column offsets of its parts (multiples of 8; the columns between are zero rows)
  int o_q = 0, o_k = 0, o_v = 0, o_lq = 0, o_lk = 0, o_lv = 0, o_g = 0, n_in = 0;
  // cache and state of the layer itself
  size_t kv_off = 0, pool_off = 0, state_off = 0;
  // weights (device)
  const bf16 *norm1 = nullptr, *norm1_b = nullptr, *norm2 = nullptr, *norm2_b = nullptr;
  const bf16 *hc1_in = nullptr, *hc1_out = nullptr, *hc1_mix = nullptr, *hc2_in = nullptr, *hc2_out = nullptr, *hc2_mix = nullptr;
  const bf16 *w_in = nullptr, *q_norm = nullptr, *k_norm = nullptr, *talk = nullptr, *wo = nullptr, *lin_norm = nullptr, *lin_wo = nullptr,
             *left_out = nullptr, *right_out = nullptr;
  const bf16 *w_gu = nullptr, *w_down = nullptr;
};
struct GbModel : RowFamily {
  const char* family_name() const override { return "gebadra"; }
  cudaError_t forward(qie_engine* e, int n, int n_seg, int n_out, int max_kv_len, float temperature, bool advance) override;
  void reset_slot(qie_engine* e, int seq) override;
  void release() override;
  size_t layer_runs() const override { return layers.size(); }

  int streams = 1;
  float eps = 1e-6f;
  std::vector<GbLayer> layers;
  const bf16 *embed = nullptr, *final_norm = nullptr, *final_norm_b = nullptr, *head = nullptr;
  bf16* blob = nullptr;
  size_t blob_bytes = 0;
  std::vector<RotaryCfg> rope_cfg;
  std::vector<float*> rope_cos, rope_sin;
  float* decay_tab = nullptr;
  // one page pool for the key/value rows and the pooled rows of every parallel layer
  void* kv_pool = nullptr;
  size_t page_elems = 0;
  // recurrent state: slot s at state + s * slot_floats
  float* state = nullptr;
  size_t slot_floats = 0;
  // activations (fp32), sized by max_batch_tokens: X streams, hn normed sublayer input, p0 projections, p1 / p2 outputs of the
  // attention and of the recurrence, p3 normed and rotated queries / feed-forward hidden rows, y1 / y2 sublayer outputs, xo normed output rows
  float *X = nullptr, *hn = nullptr, *p0 = nullptr, *p1 = nullptr, *p2 = nullptr, *p3 = nullptr, *y1 = nullptr, *y2 = nullptr, *xo = nullptr;
  TcProjector tc;
  // bf16 rows between the producers and consumers of tensor-core GEMMs
  bf16 *hb = nullptr, *mb = nullptr, *rb = nullptr, *fb = nullptr, *y1b = nullptr, *y2b = nullptr;
  float* attn_ws = nullptr;
  size_t attn_ws_floats = 0;
  float* scan_ws = nullptr;
  size_t scan_ws_floats = 0;
};

std::string gebadra_create(qie_engine* e, const std::string& dir, int* code);
std::string gebadra_create_synthetic(qie_engine* e, const std::string& cfg_json, uint64_t seed, int* code);

}  // namespace qie
