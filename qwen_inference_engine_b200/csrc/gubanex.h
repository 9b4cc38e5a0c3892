// gubanex.h -- the Gubanex model family: a decoder with one fp32 residual stream and RMS norms with zero-centred weights,
// x += mixer(norm1(x)), x += ff(norm2(x)).  A layer's mixer is one of
//  * chunked attention: grouped queries, partial rotary positions in the "rotate half" pairing with frequencies scaled by their
//    wavelength, queries and keys normed without a weight after the rotation, a softmax over the keys of the row's own chunk of positions;
//  * gated linear attention: S_t = diag(decay_t) S_(t-1) + k_t v_t^T with a decay per key channel that comes from a low-rank map of the
//    input, an fp32 state per sequence, a weighted RMS norm per head and a SiLU gate;
// and its feed-forward is a mixture of SiLU-gated experts (sigmoid router, weights that scale the experts' INPUT, not
// renormalised) or absent.  A run of consecutive layers may be repeated (a loop: the same weights, a cache or state of its own per
// pass); the embedding is added to the stream again before every pass but the first.  Logits are scaled and soft-capped.
//
// New mechanisms are options of launchers that other families use, or stand beside the ones they resemble: chunks and unit norms of the
// paged attention (attn_gqa.cu, attn_gqa_tc.cu), the gated decay of the linear attention (linear_attn.cu), zero-centred weights, the repeated
// embedding and the router's rider of the norm step (rmsnorm_f32.cu), scaled expert inputs (moe.cu, gemm_grouped.cu,
// activations.cu), frequencies scaled by wavelength (family.h).  gubanex_model.cu holds the configuration reader, the weight loader and
// the launch order.  The family shares the engine's sequences, page allocator, block tables, row metadata, sampler, scheduler and
// C ABI with the other families.
#pragma once
#include <cuda_runtime.h>

#include <string>
#include <vector>

#include "common.cuh"
#include "dedunex.h"
#include "ditenex.h"
#include "family.h"
#include "fosavik.h"
#include "gebadra.h"
#include "nogatar.h"

struct qie_engine;

namespace qie {

struct GxLayer {
  int type = 0;  // 0 attention, 1 gla
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  // attention
  int chunk = 0;  // 0: every earlier key
  float scale = 1.f;
  RotaryCfg rot;
  int rope_id = -1;
  // gla
  int rank = 0;
  float tau = 1.f;
  // feed-forward (experts 0 = none)
  int experts = 0, top = 0, ff = 0;
  // the input projection as one matrix: column offsets of its parts (multiples of 8; the columns between are zero rows)
  int o_q = 0, o_k = 0, o_v = 0, o_g = 0, o_low = 0, n_in = 0;
  // weights (device)
  const bf16 *norm1 = nullptr, *norm2 = nullptr, *w_in = nullptr, *wo = nullptr, *head_norm = nullptr, *a2 = nullptr, *a2_b = nullptr;
  const bf16 *w_router = nullptr, *w_egu = nullptr, *w_edown = nullptr;
};
// one execution of a layer: a layer inside the loop runs `times` times, each with its own cache rows or state
struct GxRun {
  int layer = 0;
  bool again = false;    // the first layer of a pass but the first: the embedding is added in front of it
  size_t kv_off = 0;     // elements into a page (attention)
  size_t state_off = 0;  // floats into a slot's state (gla)
};
struct GxModel : RowFamily {
  const char* family_name() const override { return "gubanex"; }
  cudaError_t forward(qie_engine* e, int n, int n_seg, int n_out, int max_kv_len, float temperature, bool advance) override;
  void reset_slot(qie_engine* e, int seq) override;
  void release() override;
  size_t layer_runs() const override { return runs.size(); }

  float eps = 1e-6f, embed_scale = 1.f, logit_scale = 1.f, softcap = 0.f;
  int loop_start = 0, loop_stop = 0, loop_times = 1;
  std::vector<GxLayer> layers;
  std::vector<GxRun> runs;
  const bf16 *embed = nullptr, *final_norm = nullptr, *head = nullptr;
  bf16* blob = nullptr;
  size_t blob_bytes = 0;
  std::vector<RotaryCfg> rope_cfg;
  std::vector<float*> rope_cos, rope_sin;
  // paged key/value rows of every attention run
  void* kv_pool = nullptr;
  size_t page_elems = 0;
  // recurrent state: slot s at state + s * slot_floats
  float* state = nullptr;
  size_t slot_floats = 0;
  // activations (fp32), sized by max_batch_tokens: x residual stream, hn normed sublayer input, p0 projections, p1 mixer output, p3 normed
  // and rotated queries, y projected mixer output, top_w / top_idx router choice, he / hg / ye expert rows grouped by expert, perm_w their
  // input weights, xo normed output rows
  float *x = nullptr, *hn = nullptr, *p0 = nullptr, *p1 = nullptr, *p3 = nullptr, *y = nullptr, *xo = nullptr;
  float *top_w = nullptr, *perm_w = nullptr, *he = nullptr, *hg = nullptr, *ye = nullptr;
  int *top_idx = nullptr, *grp_off = nullptr, *perm_row = nullptr, *slot_of = nullptr;
  TcProjector tc;
  // bf16 rows between the producers and consumers of tensor-core GEMMs: hb normed input, mb mixer output, yb projected mixer output, hgr
  // normed rows in the experts' order, hgb gated hidden rows of the experts, yeb their outputs
  bf16 *hb = nullptr, *mb = nullptr, *yb = nullptr, *hgr = nullptr, *hgb = nullptr, *yeb = nullptr;
  float* attn_ws = nullptr;
  size_t attn_ws_floats = 0;
  float* scan_ws = nullptr;  // chunk states of the linear attention
  size_t scan_ws_floats = 0;
  float* decay_ws = nullptr;  // running sums of its decays
};

std::string gubanex_create(qie_engine* e, const std::string& dir, int* code);
std::string gubanex_create_synthetic(qie_engine* e, const std::string& cfg_json, uint64_t seed, int* code);

}  // namespace qie
