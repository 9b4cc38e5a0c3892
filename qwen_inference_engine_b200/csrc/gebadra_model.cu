// gebadra_model.cu -- the Gebadra family on the engine: configuration reader (config.json), weight loader
// (model.safetensors -> one device blob), the page pool shared by the key/value rows and the pooled rows of the parallel
// layers, the state slots of the linear recurrences, and the launch order of one forward over a batch of rows.  A row is
// (sequence slot, position) exactly as in the other families; rows of one sequence are consecutive and in position order,
// rows of different sequences may be portions of prompts next to single decoded tokens.  Every size and constant comes
// from the configuration.  A layer with weights_of reads another layer's weights and keeps cache rows and state of its own.
#include "gebadra.h"

#include <math.h>
#include <stdio.h>
#include <string.h>

#include <algorithm>
#include <map>

#include "engine.h"
#include "json_min.h"
#include "launch.h"

namespace qie {
namespace {

#define NEED(cond, msg)      \
  do {                       \
    if (!(cond)) return msg; \
  } while (0)

int as_int(const JsonValue* v, int dflt) { return v && v->is_number() ? (int)llround(v->num) : dflt; }
int up8(int v) { return (v + 7) & ~7; }

std::string parse_linear(const JsonValue& mx, GbLinear* l) {
  l->heads = as_int(mx.have("heads"), 0);
  l->dim = as_int(mx.have("dim"), 0);
  l->vdim = as_int(mx.have("vdim"), l->dim);
  NEED(l->heads > 0 && l->dim > 0 && l->vdim > 0, "config.json: heads / dim / vdim of a linear recurrence missing");
  NEED(l->dim <= 256, "config.json: dim of a linear recurrence above 256");
  const JsonValue* dc = mx.have("decay");
  NEED(dc && dc->kind == JsonValue::Array && (int)dc->arr.size() == l->heads, "config.json: decay must list one number per head");
  for (const JsonValue& d : dc->arr) {
    NEED(d.is_number(), "config.json: decay must be numbers");
    l->decay.push_back(d.num);
  }
  return "";
}

std::string parse_attention(const JsonValue& mx, GbLayer* L) {
  L->heads = as_int(mx.have("heads"), 0);
  L->kv_heads = as_int(mx.have("kv_heads"), L->heads);
  L->dim = as_int(mx.have("dim"), 0);
  L->vdim = as_int(mx.have("vdim"), L->dim);
  NEED(L->heads > 0 && L->kv_heads > 0 && L->dim > 0 && L->vdim > 0, "config.json: attention heads / kv_heads / dim / vdim missing");
  NEED(L->heads % L->kv_heads == 0, "config.json: heads must be a multiple of kv_heads");
  NEED(mx.have("scale") && mx.have("scale")->is_number(), "config.json: attention without scale");
  L->scale = (float)mx.have("scale")->num;
  const JsonValue* mk = mx.have("mask");
  NEED(mk, "config.json: attention without mask");
  L->window = as_int(mk->have("size"), 0), L->pool = as_int(mk->have("pool"), 0);
  NEED(L->window > 0 && L->pool > 0, "config.json: mask.size and mask.pool must be positive");
  if (const JsonValue* rt = mx.have("rot")) {
    L->rot.dims = as_int(rt->have("dims"), 0);
    NEED(L->rot.dims >= 0 && L->rot.dims % 2 == 0 && L->rot.dims <= L->dim, "config.json: rot.dims must be even and at most the head size");
    L->rot.base = rt->have("base") ? rt->have("base")->num : 10000.0;
    NEED(L->rot.base > 0.0, "config.json: rot.base");
    if (const JsonValue* sc = rt->have("scaling")) {
      L->rot.linear = sc->have("factor") ? sc->have("factor")->num : 1.0;
      NEED(L->rot.linear > 0.0, "config.json: rot.scaling.factor");
    }
  }
  return "";
}

std::string parse_config(const JsonValue& root, GbModel* m) {
  NEED(root.kind == JsonValue::Object, "config.json: not an object");
  m->vocab = as_int(root.have("vocab"), 0);
  m->width = as_int(root.have("width"), 0);
  NEED(m->vocab > 0 && m->width > 0, "config.json: vocab / width missing");
  m->streams = as_int(root.have("streams"), 1);
  NEED(m->streams >= 1 && m->streams <= 8, "config.json: streams must be 1 to 8");
  if (const JsonValue* nm = root.have("norm"))
    if (nm->have("eps") && nm->have("eps")->is_number()) m->eps = (float)nm->have("eps")->num;
  const JsonValue* layers = root.have("layers");
  NEED(layers && layers->kind == JsonValue::Array && !layers->arr.empty(), "config.json: layers missing");
  for (const JsonValue& jl : layers->arr) {
    GbLayer L;
    const JsonValue* type = jl.have("type");
    const JsonValue* mx = jl.have("mixer");
    NEED(type && type->kind == JsonValue::String && mx && mx->kind == JsonValue::Object, "config.json: layer without type / mixer");
    std::string err;
    if (type->str == "lightning") {
      L.type = 0;
      err = parse_linear(*mx, &L.lin);
    } else if (type->str == "parallel") {
      L.type = 1;
      const JsonValue *lf = mx->have("left"), *rt = mx->have("right");
      NEED(lf && rt, "config.json: parallel mixer without left / right");
      err = parse_attention(*lf, &L);
      if (err.empty()) err = parse_linear(*rt, &L.lin);
    } else {
      return "config.json: unknown layer type '" + type->str + "'";
    }
    if (!err.empty()) return err;
    if (const JsonValue* mlp = jl.have("mlp")) {
      if (mlp->kind == JsonValue::Object) {
        const JsonValue* kind = mlp->have("kind");
        NEED(kind && kind->kind == JsonValue::String && kind->str == "dense", "config.json: mlp.kind must be dense");
        L.ff = as_int(mlp->have("ff"), 0);
        NEED(L.ff > 0, "config.json: dense mlp without ff");
      }
    }
    const JsonValue* wf = jl.have("weights_of");
    if (wf && wf->is_number()) L.weights_of = as_int(wf, -1);
    // the parts of the input projection, each starting at a multiple of 8 columns
    int at = 0;
    auto part = [&](int n) {
      const int o = at;
      at += up8(n);
      return o;
    };
    if (L.type == 1) L.o_q = part(L.heads * L.dim), L.o_k = part(L.kv_heads * L.dim), L.o_v = part(L.kv_heads * L.vdim);
    const int nk = L.lin.heads * L.lin.dim, nv = L.lin.heads * L.lin.vdim;
    L.o_lq = part(nk), L.o_lk = part(nk), L.o_lv = part(nv), L.o_g = part(nv);
    L.n_in = at;
    m->layers.push_back(L);
  }
  // a layer that uses another one's weights: follow to the layer that has tensors; the entries must describe the same sizes
  const int NL = (int)m->layers.size();
  for (int i = 0; i < NL; ++i) {
    GbLayer& L = m->layers[i];
    int j = i, steps = 0;
    while (m->layers[j].weights_of >= 0) {
      j = m->layers[j].weights_of;
      NEED(j < NL && ++steps <= NL, "config.json: weights_of does not lead to a layer with tensors");
    }
    if (j == i) continue;
    const GbLayer& O = m->layers[j];
    NEED(O.type == L.type && O.n_in == L.n_in && O.ff == L.ff && O.heads == L.heads && O.kv_heads == L.kv_heads && O.dim == L.dim && O.vdim == L.vdim &&
             O.lin.heads == L.lin.heads && O.lin.dim == L.lin.dim && O.lin.vdim == L.lin.vdim,
         "config.json: a layer with weights_of must have the sizes of that layer");
  }
  for (int i = 0; i < NL; ++i)
    while (m->layers[i].weights_of >= 0 && m->layers[m->layers[i].weights_of].weights_of >= 0) m->layers[i].weights_of = m->layers[m->layers[i].weights_of].weights_of;
  return "";
}

// tensors in blob order; a layer's input projections are ONE matrix (one GEMM of the normed input), so are the
// feed-forward's gate and up; the parts of the former start at multiples of 8 rows, the rows between them stay zero (kind 3:
// not in the file)
std::vector<TensorSpec> build_layout(const GbModel& m) {
  BlobLayout bl;
  auto pad = [&]() { bl.pad(); };
  auto add = [&](const std::string& name, size_t rows, size_t cols, int kind) { bl.add(name, rows, cols, kind); };
  const size_t W = m.width, S = m.streams;
  pad(), add("embed", m.vocab, W, 0);
  for (size_t i = 0; i < m.layers.size(); ++i) {
    const GbLayer& L = m.layers[i];
    if (L.weights_of >= 0) continue;
    const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.", lp = L.type == 1 ? mp + "right." : mp;
    int at = 0;
    auto part = [&](const std::string& name, int rows, int off) {  // zero rows up to the part's offset, then the part
      if (off > at) add(p + "zero" + std::to_string(off), off - at, W, 3);
      add(name, rows, W, 0);
      at = off + rows;
    };
    pad(), add(p + "norm1", W, 0, 1);
    pad(), add(p + "norm1.b", W, 0, 2);
    pad(), add(p + "hc1.in", S, 0, 1);
    pad(), add(p + "hc1.out", S, 0, 1);
    pad(), add(p + "hc1.mix", S, S, 0);
    pad();
    if (L.type == 1) part(mp + "left.q", L.heads * L.dim, L.o_q), part(mp + "left.k", L.kv_heads * L.dim, L.o_k), part(mp + "left.v", L.kv_heads * L.vdim, L.o_v);
    const int nk = L.lin.heads * L.lin.dim, nv = L.lin.heads * L.lin.vdim;
    part(lp + "q", nk, L.o_lq), part(lp + "k", nk, L.o_lk), part(lp + "v", nv, L.o_lv), part(lp + "g", nv, L.o_g);
    if (L.n_in > at) add(p + "zero" + std::to_string(L.n_in), L.n_in - at, W, 3);
    if (L.type == 1) {
      pad(), add(mp + "left.q.norm", (size_t)L.heads * L.dim, 0, 1);
      pad(), add(mp + "left.k.norm", (size_t)L.kv_heads * L.dim, 0, 1);
      pad(), add(mp + "left.talk", L.heads, L.heads, 0);
      pad(), add(mp + "left.o", W, (size_t)L.heads * L.vdim, 0);
      pad(), add(mp + "left.out", W, 0, 1);
      pad(), add(mp + "right.out", W, 0, 1);
    } else {
      pad(), add(mp + "norm", nv, 0, 1);
    }
    pad(), add(lp + "o", W, nv, 0);
    if (L.ff > 0) {
      pad(), add(p + "norm2", W, 0, 1);
      pad(), add(p + "norm2.b", W, 0, 2);
      pad(), add(p + "hc2.in", S, 0, 1);
      pad(), add(p + "hc2.out", S, 0, 1);
      pad(), add(p + "hc2.mix", S, S, 0);
      pad(), add(p + "mlp.gate", L.ff, W, 0), add(p + "mlp.up", L.ff, W, 0);
      pad(), add(p + "mlp.down", W, L.ff, 0);
    }
  }
  pad(), add("final.norm", W, 0, 1);
  pad(), add("final.norm.b", W, 0, 2);
  pad(), add("head", m.vocab, W, 0);
  return bl.t;
}

#define CUS(expr)                                                      \
  do {                                                                 \
    cudaError_t _e = (expr);                                           \
    if (_e != cudaSuccess) {                                           \
      *code = QIE_ECUDA;                                               \
      return std::string(#expr) + ": " + cudaGetErrorString(_e);       \
    }                                                                  \
  } while (0)

std::string finish_setup(qie_engine* e, const std::vector<TensorSpec>& t, const std::vector<uint16_t>& blob, int* code) {
  GbModel* m = e->gb;
  const qie_engine_opts& o = e->opts;
  m->f32 = o.compute_dtype == QIE_DTYPE_F32;
  m->blob_bytes = blob.size() * 2;
  CUS(cudaMalloc(&m->blob, m->blob_bytes));
  CUS(cudaMemcpy(m->blob, blob.data(), m->blob_bytes, cudaMemcpyHostToDevice));
  std::map<std::string, const TensorSpec*> at;
  for (const TensorSpec& s : t) at[s.name] = &s;
  auto P = [&](const std::string& n) -> const bf16* {
    auto it = at.find(n);
    return it == at.end() ? nullptr : m->blob + it->second->off;
  };
  m->embed = P("embed"), m->final_norm = P("final.norm"), m->final_norm_b = P("final.norm.b"), m->head = P("head");
  e->cfg = qie_config{m->width, 0, (int)m->layers.size(), 0, 0, 0, m->vocab, o.context};
  const size_t W = m->width, R = o.max_batch_tokens;
  size_t w0 = 1, w1 = 1, w2 = 1, w3 = 1, wff = 1, hmv = 1, maxk = W, maxn = W, scan = 1;
  std::vector<float> powers;
  std::vector<size_t> pow_at;
  // cache rows, pooled rows and state of every layer: a page holds page_size positions and the pooled rows of the blocks that end
  // in it, every layer's rows starting at a multiple of 8 elements
  size_t page_elems = 0, slot_floats = 0;
  for (size_t i = 0; i < m->layers.size(); ++i) {
    GbLayer& L = m->layers[i];
    const std::string p = "l" + std::to_string(L.weights_of >= 0 ? L.weights_of : (int)i) + ".", mp = p + "mix.", lp = L.type == 1 ? mp + "right." : mp;
    L.norm1 = P(p + "norm1"), L.norm1_b = P(p + "norm1.b"), L.norm2 = P(p + "norm2"), L.norm2_b = P(p + "norm2.b");
    L.hc1_in = P(p + "hc1.in"), L.hc1_out = P(p + "hc1.out"), L.hc1_mix = P(p + "hc1.mix");
    L.hc2_in = P(p + "hc2.in"), L.hc2_out = P(p + "hc2.out"), L.hc2_mix = P(p + "hc2.mix");
    L.w_in = P(L.type == 1 ? mp + "left.q" : mp + "q");
    L.lin_norm = P(mp + "norm"), L.lin_wo = P(lp + "o");
    L.w_gu = P(p + "mlp.gate"), L.w_down = P(p + "mlp.down");
    const size_t nv = (size_t)L.lin.heads * L.lin.vdim;
    w0 = std::max(w0, (size_t)L.n_in), maxn = std::max(maxn, (size_t)L.n_in);
    w2 = std::max(w2, nv), maxk = std::max(maxk, nv);
    scan = std::max(scan, linear_ws_floats(R, (size_t)o.max_seqs, L.lin.heads, L.lin.dim, L.lin.vdim));
    if (L.ff > 0) {
      w0 = std::max(w0, (size_t)2 * L.ff), maxn = std::max(maxn, (size_t)2 * L.ff);
      wff = std::max(wff, (size_t)L.ff), maxk = std::max(maxk, (size_t)L.ff);
    }
    L.state_off = slot_floats, slot_floats += (nv * L.lin.dim + 3) / 4 * 4;
    pow_at.push_back(powers.size());
    for (double d : L.lin.decay) {
      double x = 1.0;
      for (int k = 0; k <= LINEAR_CHUNK; ++k, x *= d) powers.push_back((float)x);
    }
    if (L.type == 1) {
      const size_t H = L.heads, G = L.kv_heads, row = G * L.dim + G * L.vdim;
      L.q_norm = P(mp + "left.q.norm"), L.k_norm = P(mp + "left.k.norm"), L.talk = P(mp + "left.talk"), L.wo = P(mp + "left.o");
      L.left_out = P(mp + "left.out"), L.right_out = P(mp + "right.out");
      w1 = std::max(w1, H * L.vdim), w3 = std::max(w3, H * L.dim), maxk = std::max(maxk, H * L.vdim);
      hmv = std::max(hmv, gqa_ws_floats(1, L.heads, 1, L.kv_heads * L.vdim));
      L.kv_off = page_elems, page_elems += ((size_t)o.page_size * row + 7) / 8 * 8;
      L.pool_off = page_elems, page_elems += ((size_t)kv_pool_rows(o.page_size, L.pool) * row + 7) / 8 * 8;
      if (L.rot.dims > 0) {
        size_t id = 0;
        while (id < m->rope_cfg.size() && !(m->rope_cfg[id] == L.rot)) ++id;
        if (id == m->rope_cfg.size()) m->rope_cfg.push_back(L.rot);
        L.rope_id = (int)id;
      }
    }
  }
  CUS(cudaMalloc(&m->decay_tab, powers.size() * sizeof(float)));
  CUS(cudaMemcpy(m->decay_tab, powers.data(), powers.size() * sizeof(float), cudaMemcpyHostToDevice));
  for (size_t i = 0; i < m->layers.size(); ++i) m->layers[i].lin.decay_pow = m->decay_tab + pow_at[i];
  for (const RotaryCfg& r : m->rope_cfg) {
    std::vector<float> c, s;
    rotary_tables(r, o.context, &c, &s);
    float *cd = nullptr, *sd = nullptr;
    CUS(cudaMalloc(&cd, std::max<size_t>(c.size(), 1) * sizeof(float)));
    m->rope_cos.push_back(cd);
    CUS(cudaMalloc(&sd, std::max<size_t>(s.size(), 1) * sizeof(float)));
    m->rope_sin.push_back(sd);
    CUS(cudaMemcpy(cd, c.data(), c.size() * sizeof(float), cudaMemcpyHostToDevice));
    CUS(cudaMemcpy(sd, s.data(), s.size() * sizeof(float), cudaMemcpyHostToDevice));
  }
  m->page_elems = page_elems;
  const size_t elt = m->f32 ? 4 : 2;
  const size_t page_bytes = std::max<size_t>(page_elems * elt, 16);
  int n_pages = o.max_pages;
  if (n_pages <= 0) n_pages = (int)std::max<size_t>(1, (o.kv_bytes ? o.kv_bytes : ((size_t)1 << 30)) / page_bytes);
  CUS(cudaMalloc(&m->kv_pool, (size_t)n_pages * page_bytes));
  CUS(cudaMemsetAsync(m->kv_pool, 0, (size_t)n_pages * page_bytes, e->stream));
  e->kv = KvGeom{nullptr, n_pages, o.page_size, (int)m->layers.size(), 1, 0};
  CUS(engine_alloc_shared(e, n_pages, o.context));
  m->slot_floats = std::max<size_t>(slot_floats, 4);
  CUS(cudaMalloc(&m->state, (size_t)o.max_seqs * m->slot_floats * sizeof(float)));
  CUS(cudaMemsetAsync(m->state, 0, (size_t)o.max_seqs * m->slot_floats * sizeof(float), e->stream));
  // activations
  auto fbuf = [&](float** p, size_t n) { return cudaMalloc(p, std::max<size_t>(n, 4) * sizeof(float)); };
  CUS(fbuf(&m->X, R * m->streams * W));
  CUS(fbuf(&m->hn, R * W));
  CUS(fbuf(&m->p0, R * w0));
  CUS(fbuf(&m->p1, R * w1));
  CUS(fbuf(&m->p2, R * w2));
  CUS(fbuf(&m->p3, R * std::max(w3, wff)));
  CUS(fbuf(&m->y1, R * W));
  CUS(fbuf(&m->y2, R * W));
  CUS(fbuf(&m->xo, R * W));
  m->attn_ws_floats = (R + 2048) * hmv;  // room for key splits when a step has few rows
  CUS(fbuf(&m->attn_ws, m->attn_ws_floats));
  if (!m->f32) {
    m->scan_ws_floats = scan;
    CUS(fbuf(&m->scan_ws, m->scan_ws_floats));
    CUS(m->tc.alloc(R, maxk, std::max(maxn, (size_t)m->vocab), e->stream));
    auto bbuf = [&](bf16** p, size_t n) { return cudaMalloc(p, std::max<size_t>(n, 8) * sizeof(bf16)); };
    CUS(bbuf(&m->hb, R * W));
    CUS(bbuf(&m->mb, R * w1));
    CUS(bbuf(&m->rb, R * w2));
    CUS(bbuf(&m->fb, R * wff));
    CUS(bbuf(&m->y1b, R * W));
    CUS(bbuf(&m->y2b, R * W));
  }
  CUS(m->alloc_row_buffers(R));
  e->logits_rows = (int)R;
  CUS(cudaStreamSynchronize(e->stream));
  return "";
}

std::string create_common(qie_engine* e, const std::string& cfg_text, const std::string* st_path, uint64_t seed, int* code) {
  *code = QIE_EIO;
  JsonValue root;
  std::string err;
  if (!JsonReader::parse(cfg_text.data(), cfg_text.data() + cfg_text.size(), &root, &err)) return "config.json: " + err;
  e->gb = new GbModel();
  e->fam = e->gb;
  err = parse_config(root, e->gb);
  if (!err.empty()) return err;
  const std::vector<TensorSpec> t = build_layout(*e->gb);
  std::vector<uint16_t> blob(t.empty() ? 0 : t.back().off + t.back().elems(), 0);
  if (st_path) {
    err = load_safetensors_blob(*st_path, t, &blob);
    if (!err.empty()) return err;
  } else {
    fill_synthetic_blob(t, seed, &blob);
  }
  return finish_setup(e, t, blob, code);
}

}  // namespace

std::string gebadra_create(qie_engine* e, const std::string& dir, int* code) {
  std::string cfg;
  *code = QIE_EIO;
  if (!read_text_file(dir + "/config.json", &cfg)) return "cannot read " + dir + "/config.json";
  const std::string st = dir + "/model.safetensors";
  return create_common(e, cfg, &st, 0, code);
}

std::string gebadra_create_synthetic(qie_engine* e, const std::string& cfg_json, uint64_t seed, int* code) {
  return create_common(e, cfg_json, nullptr, seed, code);
}

void GbModel::release() {
  void* dev[] = {blob, decay_tab, kv_pool, state, X, hn, p0, p1, p2, p3, y1, y2, xo, attn_ws, scan_ws, hb, mb, rb, fb, y1b, y2b};
  tc.release();
  release_row_buffers();
  for (void* p : dev)
    if (p) cudaFree(p);
  for (float* p : rope_cos)
    if (p) cudaFree(p);
  for (float* p : rope_sin)
    if (p) cudaFree(p);
}

void GbModel::reset_slot(qie_engine* e, int seq) {
  if (state) cudaMemsetAsync(state + (size_t)seq * slot_floats, 0, slot_floats * sizeof(float), e->stream);
}

cudaError_t GbModel::forward(qie_engine* e, int n, int n_seg, int n_out, int max_kv_len, float temperature, bool advance) {
  GbModel* m = this;
  cudaStream_t st = e->stream;
  const int W = m->width, S = m->streams;
  const int rnd = m->f32 ? 0 : 1;  // bf16 serving precision: the operands of the projections are bf16 values
  const int* segs = advance ? m->iota : m->seg_start;
  const int* seg_sl = advance ? e->slot_d : m->seg_slot;
  const int* outs = advance ? m->iota : m->out_rows;
  const size_t R = e->opts.max_batch_tokens;
  // plain projection C[rows, N] = A[rows, K] Wt[N, K]^T on the fp32-accumulate kernels (tensor cores on bf16 operands,
  // plain fp32 in 32-bit mode, a warp-per-column GEMV for a decode step)
  auto proj = [&](const float* A, int lda, const bf16* Wt, int K, int N, float* C, int ldc, int rows) {
    GemmF32 g;
    g.A = A, g.lda = lda, g.W = Wt, g.ldw = K, g.C = C, g.ldc = ldc, g.M = rows, g.N = N, g.K = K, g.round_a = rnd;
    return launch_gemm_f32(g, st);
  };
  // bf16 precision and a GEMM the tcgen05 kernel takes: its producer writes bf16 rows and its consumer reads them
  auto tcfit = [&](int K, int N, const bf16* Wt) { return !m->f32 && m->tc.fits(n, K, N, Wt); };
  if (m->dump_layers && !m->layer_dump)
    if (cudaMalloc(&m->layer_dump, m->layers.size() * R * W * sizeof(float)) != cudaSuccess) return cudaErrorMemoryAllocation;
  // the read half of the next sublayer: its weights, and bf16 rows where its projection takes them
  auto read = [&](HyperStep& hs, const bf16* in, const bf16* w, const bf16* b, bool to_bf) {
    hs.in = in, hs.w = w, hs.b = b;
    if (to_bf) hs.h_bf = m->hb;
    else hs.h = m->hn;
  };
  auto step = [&]() {
    HyperStep hs;
    hs.X = m->X, hs.width = W, hs.streams = S, hs.n = n, hs.eps = m->eps;
    return hs;
  };
  auto in_fits = [&](const GbLayer& L) { return tcfit(W, L.n_in, L.w_in); };
  {
    HyperStep hs = step();
    hs.ids = e->ids_d, hs.embed = m->embed;
    const GbLayer& L = m->layers[0];
    read(hs, L.hc1_in, L.norm1, L.norm1_b, in_fits(L));
    FAM_TRY(KK_HYPER, launch_hyper_step(hs, st));
  }
  for (size_t li = 0; li < m->layers.size(); ++li) {
    const GbLayer& L = m->layers[li];
    const GbLinear& N = L.lin;
    const int ld = L.n_in, nv = N.heads * N.vdim;
    const bool tc_in = in_fits(L);
    const bf16* pb = m->tc.cb;  // the projection's result as bf16 rows
    if (tc_in) FAM_TRY(KK_F32_PROJ, m->tc.gemm_bf16(e, m->hb, L.w_in, W, L.n_in, m->tc.cb, n));
    else FAM_TRY(KK_F32_PROJ, proj(m->hn, W, L.w_in, W, L.n_in, m->p0, ld, n));
    // linear recurrence and the norm and gate behind it -> rows rb (bf16) or p2 (fp32)
    const bool tc_lo = tcfit(nv, W, L.lin_wo);
    {
      LinearAttnArgs a;
      if (tc_in) a.q_bf = pb + L.o_lq, a.k_bf = pb + L.o_lk, a.v_bf = pb + L.o_lv, a.g_bf = pb + L.o_g, a.ld_bf = ld;
      else a.q = m->p0 + L.o_lq, a.k = m->p0 + L.o_lk, a.v = m->p0 + L.o_lv, a.ld = ld;
      a.act = L.type == 0, a.k_scale = L.type == 0 ? 1.0f : 1.0f / sqrtf((float)N.dim);
      a.heads = N.heads, a.dim = N.dim, a.vdim = N.vdim, a.decay_pow = N.decay_pow, a.eps = m->eps;
      a.out = m->p2, a.ldo = nv;
      a.state = m->state + L.state_off, a.slot_stride = m->slot_floats;
      a.seg_start = segs, a.seg_slot = seg_sl, a.n_seg = n_seg, a.n_rows = n;
      a.ws = m->scan_ws, a.ws_floats = m->scan_ws_floats;
      // retention's norm covers one head, which a chunk's CTA holds whole
      const bool fused = L.type == 1 && tc_lo && linear_attention_norm_fits(a);
      if (fused) a.norm_gate = 1, a.out_bf = m->rb, a.ldo_bf = nv;
      int nl = 0;
      FAM_TRY(KK_LINEAR_ATTN, launch_linear_attention(a, st, &nl));
      e->launches += nl > 0 ? nl - 1 : 0;
      if (!fused) {
        NormGate g;
        g.v = m->p2, g.ldv = nv, g.width = nv, g.n = n, g.eps = m->eps;
        if (L.type == 0) g.w = L.lin_norm, g.groups = 1, g.act = 1;
        else g.groups = N.heads, g.act = 0;
        if (tc_in) g.g_bf = pb + L.o_g, g.ldg_bf = ld;
        else g.g = m->p0 + L.o_g, g.ldg = ld;
        if (tc_lo) g.out_bf = m->rb, g.ldo_bf = nv;
        else g.out = m->p2, g.ldo = nv;
        FAM_TRY(KK_NORM_GATE, launch_norm_gate(g, st));
      }
    }
    HyperStep hs = step();
    hs.mix = L.hc1_mix, hs.out = L.hc1_out;
    if (L.type == 1) {
      const int H = L.heads, G = L.kv_heads, d = L.dim, vd = L.vdim;
      KvRowCache c;
      c.pool = m->kv_pool, c.elt_bytes = m->f32 ? 4 : 2, c.page_size = e->kv.page_size, c.page_elems = m->page_elems;
      c.layer_off = L.kv_off, c.kw = G * d, c.vw = G * vd, c.block = L.pool, c.pool_off = L.pool_off, c.n_pages = e->kv.n_pages;
      const float* q = m->p0 + L.o_q;
      int ldq = ld;
      {  // keys (norm over all kv heads, rotation) and values -> cache rows; the queries alike
        KvStoreArgs ks;
        ks.c = c, ks.whole_norm = 1, ks.one_each = n == n_seg, ks.k_norm = L.k_norm, ks.q_norm = L.q_norm, ks.norm_dim = d, ks.eps = m->eps;
        ks.q_heads = H;
        if (tc_in) {
          ks.q_bf = pb + L.o_q, ks.k_bf = pb + L.o_k, ks.v_bf = pb + L.o_v, ks.ld_bf = ld;
          ks.q = m->p3, ks.ldq = H * d, q = m->p3, ldq = H * d;
        } else {
          ks.k = m->p0 + L.o_k, ks.ldk = ld, ks.v = m->p0 + L.o_v, ks.ldv = ld, ks.q = m->p0 + L.o_q, ks.ldq = ld;
        }
        if (L.rope_id >= 0) ks.rope = RopeTable{m->rope_cos[L.rope_id], m->rope_sin[L.rope_id], L.rot.dims, 0};
        ks.pos = e->pos_d, ks.slot = e->slot_d, ks.block_table = e->block_table_d, ks.max_pages = e->max_pages_per_seq, ks.n = n;
        FAM_TRY(KK_KV_STORE, launch_kv_store_rows(ks, st));
        if (n != n_seg) FAM_TRY(KK_KV_STORE, launch_kv_pool_rows(c, e->pos_d, e->slot_d, e->block_table_d, e->max_pages_per_seq, n, st));
      }
      const bool tc_o = tcfit(H * vd, W, L.wo);
      GqaAttnArgs g;
      g.c = c, g.q = q, g.ldq = ldq, g.out = m->p1, g.ldo = H * vd;
      if (tc_o) g.out_bf = m->mb, g.ldo_bf = H * vd;
      g.heads = H, g.kv_heads = G, g.dim = d, g.vdim = vd, g.scale = L.scale, g.window = L.window, g.talk = L.talk, g.eps = m->eps;
      g.pos = e->pos_d, g.slot = e->slot_d, g.block_table = e->block_table_d, g.max_pages = e->max_pages_per_seq, g.n = n, g.max_keys = max_kv_len;
      g.ws = m->attn_ws, g.ws_floats = m->attn_ws_floats, g.num_sms = e->num_sms;
      g.seg_start = segs, g.seg_slot = seg_sl, g.n_seg = n_seg;
      int nl = 0;
      FAM_TRY(KK_GQA_ATTN, launch_gqa_attention(g, st, &nl));
      e->launches += nl > 0 ? nl - 1 : 0;
      if (tc_o) {
        FAM_TRY(KK_F32_PROJ, m->tc.gemm_bf16(e, m->mb, L.wo, H * vd, W, m->y1b, n));
        hs.y1_bf = m->y1b;
      } else {
        FAM_TRY(KK_F32_PROJ, proj(m->p1, H * vd, L.wo, H * vd, W, m->y1, W, n));
        hs.y1 = m->y1;
      }
      if (tc_lo) {
        FAM_TRY(KK_F32_PROJ, m->tc.gemm_bf16(e, m->rb, L.lin_wo, nv, W, m->y2b, n));
        hs.y2_bf = m->y2b;
      } else {
        FAM_TRY(KK_F32_PROJ, proj(m->p2, nv, L.lin_wo, nv, W, m->y2, W, n));
        hs.y2 = m->y2;
      }
      hs.y1_norm = L.left_out, hs.y2_norm = L.right_out, hs.s1 = hs.s2 = 0.5f;
    } else if (tc_lo) {
      FAM_TRY(KK_F32_PROJ, m->tc.gemm_bf16(e, m->rb, L.lin_wo, nv, W, m->y1b, n));
      hs.y1_bf = m->y1b;
    } else {
      FAM_TRY(KK_F32_PROJ, proj(m->p2, nv, L.lin_wo, nv, W, m->y1, W, n));
      hs.y1 = m->y1;
    }
    const GbLayer* next = li + 1 < m->layers.size() ? &m->layers[li + 1] : nullptr;
    float* dump = m->dump_layers ? m->layer_dump + li * R * W : nullptr;
    auto read_next = [&](HyperStep& h) {
      if (next) read(h, next->hc1_in, next->norm1, next->norm1_b, in_fits(*next));
      h.dump = dump;
    };
    const bool tc_gu = L.ff > 0 && tcfit(W, 2 * L.ff, L.w_gu);
    if (L.ff > 0) read(hs, L.hc2_in, L.norm2, L.norm2_b, tc_gu);
    else read_next(hs);
    FAM_TRY(KK_HYPER, launch_hyper_step(hs, st));  // the mixer's write; the same launch reads for the next sublayer
    if (L.ff > 0) {
      GatedAct ga;
      ga.ff = L.ff, ga.act = 0, ga.n = n;
      if (tc_gu) {
        FAM_TRY(KK_F32_PROJ, m->tc.gemm_bf16(e, m->hb, L.w_gu, W, 2 * L.ff, m->tc.cb, n));
        ga.g_bf = m->tc.cb, ga.u_bf = m->tc.cb + L.ff, ga.ld_bf = 2 * L.ff;
      } else {
        FAM_TRY(KK_F32_PROJ, proj(m->hn, W, L.w_gu, W, 2 * L.ff, m->p0, 2 * L.ff, n));
        ga.g = m->p0, ga.u = m->p0 + L.ff, ga.ld = 2 * L.ff;
      }
      HyperStep h2 = step();
      h2.mix = L.hc2_mix, h2.out = L.hc2_out;
      if (tcfit(L.ff, W, L.w_down)) {
        ga.out_bf = m->fb, ga.ldo_bf = L.ff;
        FAM_TRY(KK_GLU, launch_gated_act(ga, st));
        FAM_TRY(KK_F32_PROJ, m->tc.gemm_bf16(e, m->fb, L.w_down, L.ff, W, m->y1b, n));
        h2.y1_bf = m->y1b;
      } else {
        ga.out = m->p3, ga.ldo = L.ff;
        FAM_TRY(KK_GLU, launch_gated_act(ga, st));
        FAM_TRY(KK_F32_PROJ, proj(m->p3, L.ff, L.w_down, L.ff, W, m->y1, W, n));
        h2.y1 = m->y1;
      }
      read_next(h2);
      FAM_TRY(KK_HYPER, launch_hyper_step(h2, st));
    }
  }
  if (n_out <= 0) return cudaSuccess;
  {
    HyperStep hs = step();
    hs.n = n_out, hs.w = m->final_norm, hs.b = m->final_norm_b, hs.h = m->xo, hs.gather = outs;
    FAM_TRY(KK_F32_NORM, launch_hyper_step(hs, st));
  }
  {
    GemmF32 g;
    g.A = m->xo, g.lda = W, g.W = m->head, g.ldw = W, g.C = m->logits, g.ldc = m->vocab, g.M = n_out, g.N = m->vocab, g.K = W, g.round_a = rnd;
    FAM_TRY(KK_LM_HEAD, launch_gemm_f32(g, st));
  }
  return sample_rows(e, n_out, temperature, advance);
}

}  // namespace qie
