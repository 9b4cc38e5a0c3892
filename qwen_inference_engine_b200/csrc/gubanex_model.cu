// gubanex_model.cu -- the Gubanex family on the engine: configuration reader (config.json), weight loader (model.safetensors -> one
// device blob), the page pool of the key/value rows of every attention run, the state slots of the gated linear attention, and the launch
// order of one forward over a batch of rows.  A row is (sequence slot, position) exactly as in the other families; rows of one sequence
// are consecutive and in position order, rows of different sequences may be portions of prompts next to single decoded tokens.  Every
// size and constant comes from the configuration or from a tensor's shape.  A layer inside the loop appears once per pass in `runs`, with
// cache rows or a state of its own.
#include "gubanex.h"

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
float as_float(const JsonValue* v, float dflt) { return v && v->is_number() ? (float)v->num : dflt; }
int up8(int v) { return (v + 7) & ~7; }

std::string parse_rot(const JsonValue* rt, int dim, RotaryCfg* r) {
  if (!rt) return "";  // no rotation
  r->dims = as_int(rt->have("dims"), 0);
  NEED(r->dims >= 0 && r->dims % 2 == 0 && r->dims <= dim, "config.json: rot.dims must be even and at most the head size");
  r->base = rt->have("base") ? rt->have("base")->number_or(10000.0) : 10000.0;
  NEED(r->base > 0.0, "config.json: rot.base");
  if (const JsonValue* sc = rt->have("scaling")) {
    auto num = [&](const char* k) { return sc->have(k) ? sc->have(k)->number_or(0.0) : 0.0; };
    r->by_wave = true;
    r->factor = num("factor"), r->original = num("original"), r->low = num("low"), r->high = num("high");
    NEED(r->factor > 0.0 && r->original > 0.0 && r->low > 0.0 && r->high >= r->low, "config.json: rot.scaling needs factor, original, low, high");
  }
  return "";
}

std::string parse_config(const JsonValue& root, GxModel* m) {
  NEED(root.kind == JsonValue::Object, "config.json: not an object");
  m->vocab = as_int(root.have("vocab"), 0);
  m->width = as_int(root.have("width"), 0);
  NEED(m->vocab > 0 && m->width > 0, "config.json: vocab / width missing");
  if (const JsonValue* nm = root.have("norm")) m->eps = as_float(nm->have("eps"), 1e-6f);
  if (const JsonValue* em = root.have("embedding")) m->embed_scale = as_float(em->have("scale"), 1.0f);
  m->logit_scale = as_float(root.have("logit_scale"), 1.0f);
  m->softcap = as_float(root.have("logit_softcap"), 0.0f);
  const JsonValue* layers = root.have("layers");
  NEED(layers && layers->kind == JsonValue::Array && !layers->arr.empty(), "config.json: layers missing");
  for (const JsonValue& jl : layers->arr) {
    GxLayer L;
    const JsonValue* type = jl.have("type");
    const JsonValue* mx = jl.have("mixer");
    NEED(type && type->kind == JsonValue::String && mx && mx->kind == JsonValue::Object, "config.json: layer without type / mixer");
    L.heads = as_int(mx->have("heads"), 0);
    L.dim = as_int(mx->have("dim"), 0);
    L.vdim = as_int(mx->have("vdim"), L.dim);
    NEED(L.heads > 0 && L.dim > 0 && L.vdim > 0, "config.json: heads / dim / vdim missing");
    if (type->str == "attention") {
      L.type = 0;
      L.kv_heads = as_int(mx->have("kv_heads"), L.heads);
      NEED(L.kv_heads > 0 && L.heads % L.kv_heads == 0, "config.json: heads must be a multiple of kv_heads");
      NEED(mx->have("scale") && mx->have("scale")->is_number(), "config.json: attention without scale");
      L.scale = (float)mx->have("scale")->num;
      if (const JsonValue* mk = mx->have("mask")) L.chunk = as_int(mk->have("size"), 0);
      NEED(L.chunk >= 0, "config.json: mask.size");
      const std::string err = parse_rot(mx->have("rot"), L.dim, &L.rot);
      if (!err.empty()) return err;
    } else if (type->str == "gla") {
      L.type = 1;
      L.tau = as_float(mx->have("tau"), 1.0f);
      NEED(L.tau > 0.f, "config.json: tau must be positive");
      NEED(L.dim <= 256, "config.json: dim of a linear recurrence above 256");
      L.rank = as_int(mx->have("rank"), 0);  // else the shape of its tensor gives it
    } else {
      return "config.json: unknown layer type '" + type->str + "'";
    }
    if (const JsonValue* mlp = jl.have("mlp")) {
      const JsonValue *kind = mlp->have("kind"), *ex = mlp->have("expert"), *rt = mlp->have("router");
      NEED(kind && kind->kind == JsonValue::String && kind->str == "moe" && ex && rt, "config.json: mlp must be of kind moe with expert / router");
      L.ff = as_int(ex->have("ff"), 0);
      L.experts = as_int(rt->have("experts"), 0);
      L.top = as_int(rt->have("top"), 0);
      NEED(L.ff > 0 && L.experts > 0 && L.top > 0 && L.top <= L.experts, "config.json: moe ff / experts / top");
    }
    m->layers.push_back(L);
  }
  const int NL = (int)m->layers.size();
  m->loop_start = m->loop_stop = 0, m->loop_times = 1;
  if (const JsonValue* lp = root.have("loop")) {
    m->loop_start = as_int(lp->have("start"), 0);
    m->loop_stop = as_int(lp->have("stop"), m->loop_start);
    m->loop_times = as_int(lp->have("times"), 1);
    NEED(m->loop_start >= 0 && m->loop_start <= m->loop_stop && m->loop_stop <= NL && m->loop_times >= 1, "config.json: loop start / stop / times");
  }
  auto run = [&](int layer, bool again) {
    GxRun r;
    r.layer = layer, r.again = again;
    m->runs.push_back(r);
  };
  for (int i = 0; i < m->loop_start; ++i) run(i, false);
  for (int t = 0; t < m->loop_times; ++t)
    for (int i = m->loop_start; i < m->loop_stop; ++i) run(i, t > 0 && i == m->loop_start);
  for (int i = m->loop_stop; i < NL; ++i) run(i, false);
  return "";
}

// the parts of every layer's input projection, each starting at a multiple of 8 columns (the ranks are known by now)
void place_parts(GxModel* m) {
  for (GxLayer& L : m->layers) {
    int at = 0;
    auto part = [&](int n) {
      const int o = at;
      at += up8(n);
      return o;
    };
    const int G = L.type == 0 ? L.kv_heads : L.heads;
    L.o_q = part(L.heads * L.dim), L.o_k = part(G * L.dim), L.o_v = part(G * L.vdim);
    if (L.type == 1) L.o_g = part(L.heads * L.vdim), L.o_low = part(L.rank);
    L.n_in = at;
  }
}

// tensors in blob order; a layer's input projections are ONE matrix (one GEMM of the normed input), so are every expert's gate and
// up; the parts of the former start at multiples of 8 rows, the rows between them stay zero (kind 3: not in the file)
std::vector<TensorSpec> build_layout(const GxModel& m) {
  BlobLayout bl;
  auto pad = [&]() { bl.pad(); };
  auto add = [&](const std::string& name, size_t rows, size_t cols, int kind) { bl.add(name, rows, cols, kind); };
  const size_t W = m.width;
  pad(), add("embed", m.vocab, W, 0);
  for (size_t i = 0; i < m.layers.size(); ++i) {
    const GxLayer& L = m.layers[i];
    const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
    int at = 0;
    auto part = [&](const std::string& name, int rows, int off) {  // zero rows up to the part's offset, then the part
      if (off > at) add(p + "zero" + std::to_string(off), off - at, W, 3);
      add(name, rows, W, 0);
      at = off + rows;
    };
    pad(), add(p + "norm1", W, 0, 4);
    pad();
    const int G = L.type == 0 ? L.kv_heads : L.heads;
    part(mp + "q", L.heads * L.dim, L.o_q), part(mp + "k", G * L.dim, L.o_k), part(mp + "v", G * L.vdim, L.o_v);
    if (L.type == 1) part(mp + "g", L.heads * L.vdim, L.o_g), part(mp + "a1", L.rank, L.o_low);
    if (L.n_in > at) add(p + "zero" + std::to_string(L.n_in), L.n_in - at, W, 3);
    if (L.type == 1) {
      pad(), add(mp + "a2", (size_t)L.heads * L.dim, L.rank, 0);
      pad(), add(mp + "a2.b", (size_t)L.heads * L.dim, 0, 2);
      pad(), add(mp + "norm", L.vdim, 0, 1);
    }
    pad(), add(mp + "o", W, (size_t)L.heads * L.vdim, 0);
    if (L.experts == 0) continue;
    pad(), add(p + "norm2", W, 0, 4);
    pad(), add(p + "mlp.router", L.experts, W, 0);
    pad();
    for (int e = 0; e < L.experts; ++e) {
      const std::string q = p + "mlp.e" + std::to_string(e) + ".";
      add(q + "gate", L.ff, W, 0), add(q + "up", L.ff, W, 0);
    }
    pad();
    for (int e = 0; e < L.experts; ++e) add(p + "mlp.e" + std::to_string(e) + ".down", W, L.ff, 0);
  }
  pad(), add("final.norm", W, 0, 4);
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
  GxModel* m = e->gx;
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
  m->embed = P("embed"), m->final_norm = P("final.norm"), m->head = P("head");
  e->cfg = qie_config{m->width, 0, (int)m->runs.size(), 0, 0, 0, m->vocab, o.context};
  const size_t W = m->width, R = o.max_batch_tokens;
  size_t w0 = 1, w1 = 1, w3 = 1, hmv = 1, maxk = W, maxn = W, scan = 1, decay = 1, w_top = 1, w_he = 1;
  int max_experts = 0;
  for (size_t i = 0; i < m->layers.size(); ++i) {
    GxLayer& L = m->layers[i];
    const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
    L.norm1 = P(p + "norm1"), L.norm2 = P(p + "norm2"), L.w_in = P(mp + "q"), L.wo = P(mp + "o");
    L.w_router = P(p + "mlp.router"), L.w_egu = P(p + "mlp.e0.gate"), L.w_edown = P(p + "mlp.e0.down");
    const size_t nv = (size_t)L.heads * L.vdim;
    w0 = std::max(w0, (size_t)L.n_in), maxn = std::max(maxn, (size_t)L.n_in);
    w1 = std::max(w1, nv), maxk = std::max(maxk, nv);
    if (L.type == 0) {
      w3 = std::max(w3, (size_t)L.heads * L.dim);
      hmv = std::max(hmv, gqa_ws_floats(1, L.heads, 1, L.vdim));
      if (L.rot.dims > 0) {
        size_t id = 0;
        while (id < m->rope_cfg.size() && !(m->rope_cfg[id] == L.rot)) ++id;
        if (id == m->rope_cfg.size()) m->rope_cfg.push_back(L.rot);
        L.rope_id = (int)id;
      }
    } else {
      L.a2 = P(mp + "a2"), L.a2_b = P(mp + "a2.b"), L.head_norm = P(mp + "norm");
      scan = std::max(scan, linear_ws_floats(R, (size_t)o.max_seqs, L.heads, L.dim, L.vdim));
      decay = std::max(decay, gated_decay_floats(R, L.heads, L.dim));
    }
    if (L.experts > 0) {
      w_top = std::max(w_top, (size_t)L.top);
      w_he = std::max(w_he, (size_t)L.top * 2 * L.ff);
      max_experts = std::max(max_experts, L.experts);
    }
  }
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
  // cache rows and state of every run: a page holds page_size positions of every attention run, each run's block of rows starting at a
  // multiple of 8 elements
  size_t page_elems = 0, slot_floats = 0;
  for (GxRun& r : m->runs) {
    const GxLayer& L = m->layers[r.layer];
    if (L.type == 0) r.kv_off = page_elems, page_elems += ((size_t)o.page_size * L.kv_heads * (L.dim + L.vdim) + 7) / 8 * 8;
    else r.state_off = slot_floats, slot_floats += ((size_t)L.heads * L.dim * L.vdim + 3) / 4 * 4;
  }
  m->page_elems = page_elems;
  const size_t elt = m->f32 ? 4 : 2;
  const size_t page_bytes = std::max<size_t>(page_elems * elt, 16);
  int n_pages = o.max_pages;
  if (n_pages <= 0) n_pages = (int)std::max<size_t>(1, (o.kv_bytes ? o.kv_bytes : ((size_t)1 << 30)) / page_bytes);
  CUS(cudaMalloc(&m->kv_pool, (size_t)n_pages * page_bytes));
  CUS(cudaMemsetAsync(m->kv_pool, 0, (size_t)n_pages * page_bytes, e->stream));
  e->kv = KvGeom{nullptr, n_pages, o.page_size, (int)m->runs.size(), 1, 0};
  CUS(engine_alloc_shared(e, n_pages, o.context));
  m->slot_floats = std::max<size_t>(slot_floats, 4);
  CUS(cudaMalloc(&m->state, (size_t)o.max_seqs * m->slot_floats * sizeof(float)));
  CUS(cudaMemsetAsync(m->state, 0, (size_t)o.max_seqs * m->slot_floats * sizeof(float), e->stream));
  // activations
  auto fbuf = [&](float** p, size_t n) { return cudaMalloc(p, std::max<size_t>(n, 4) * sizeof(float)); };
  CUS(fbuf(&m->x, R * W));
  CUS(fbuf(&m->hn, R * W));
  CUS(fbuf(&m->p0, R * w0));
  CUS(fbuf(&m->p1, R * w1));
  CUS(fbuf(&m->p3, R * w3));
  CUS(fbuf(&m->y, R * W));
  CUS(fbuf(&m->xo, R * W));
  CUS(fbuf(&m->top_w, R * w_top));
  CUS(fbuf(&m->perm_w, R * w_top));
  CUS(fbuf(&m->he, max_experts ? R * w_he : 1));
  CUS(fbuf(&m->hg, max_experts ? R * w_he / 2 : 1));
  CUS(fbuf(&m->ye, max_experts ? R * w_top * W : 1));
  CUS(cudaMalloc(&m->top_idx, R * w_top * sizeof(int)));
  CUS(cudaMalloc(&m->perm_row, R * w_top * sizeof(int)));
  CUS(cudaMalloc(&m->slot_of, R * w_top * sizeof(int)));
  CUS(cudaMalloc(&m->grp_off, ((size_t)max_experts + 2) * sizeof(int)));
  m->attn_ws_floats = (R + 2048) * hmv;  // room for key splits when a step has few rows
  CUS(fbuf(&m->attn_ws, m->attn_ws_floats));
  if (!m->f32) {
    m->scan_ws_floats = scan;
    CUS(fbuf(&m->scan_ws, m->scan_ws_floats));
    CUS(fbuf(&m->decay_ws, decay));
    CUS(m->tc.alloc(R, maxk, std::max(maxn, (size_t)m->vocab), e->stream));
    auto bbuf = [&](bf16** p, size_t n) { return cudaMalloc(p, std::max<size_t>(n, 8) * sizeof(bf16)); };
    CUS(bbuf(&m->hb, R * W));
    CUS(bbuf(&m->mb, R * w1));
    CUS(bbuf(&m->yb, R * W));
    CUS(bbuf(&m->hgr, max_experts ? R * w_top * W : 1));
    CUS(bbuf(&m->hgb, max_experts ? R * w_he / 2 : 1));
    CUS(bbuf(&m->yeb, max_experts ? R * w_top * W : 1));
  }
  CUS(m->alloc_row_buffers(R));
  e->logits_rows = (int)R;
  CUS(cudaStreamSynchronize(e->stream));
  return "";
}

constexpr int DEFAULT_RANK = 16;  // of generated weights, where the configuration names none

std::string create_common(qie_engine* e, const std::string& cfg_text, const std::string* st_path, uint64_t seed, int* code) {
  *code = QIE_EIO;
  JsonValue root;
  std::string err;
  if (!JsonReader::parse(cfg_text.data(), cfg_text.data() + cfg_text.size(), &root, &err)) return "config.json: " + err;
  e->gx = new GxModel();
  e->fam = e->gx;
  err = parse_config(root, e->gx);
  if (!err.empty()) return err;
  std::map<std::string, std::vector<size_t>> shapes;
  if (st_path) {
    err = safetensors_shapes(*st_path, &shapes);
    if (!err.empty()) return err;
  }
  for (size_t i = 0; i < e->gx->layers.size(); ++i) {  // the rank of the decays' low-rank map stands in its tensor's shape
    GxLayer& L = e->gx->layers[i];
    if (L.type != 1) continue;
    const std::string name = "l" + std::to_string(i) + ".mix.a1";
    if (!st_path) {
      if (L.rank <= 0) L.rank = DEFAULT_RANK;
      continue;
    }
    const auto it = shapes.find(name);
    if (it == shapes.end() || it->second.size() != 2 || it->second[0] == 0) return "tensor " + name + " missing or not a matrix in " + *st_path;
    L.rank = (int)it->second[0];
  }
  place_parts(e->gx);
  const std::vector<TensorSpec> t = build_layout(*e->gx);
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

std::string gubanex_create(qie_engine* e, const std::string& dir, int* code) {
  std::string cfg;
  *code = QIE_EIO;
  if (!read_text_file(dir + "/config.json", &cfg)) return "cannot read " + dir + "/config.json";
  const std::string st = dir + "/model.safetensors";
  return create_common(e, cfg, &st, 0, code);
}

std::string gubanex_create_synthetic(qie_engine* e, const std::string& cfg_json, uint64_t seed, int* code) {
  return create_common(e, cfg_json, nullptr, seed, code);
}

void GxModel::release() {
  void* dev[] = {blob, kv_pool, state, x, hn, p0, p1, p3, y, xo, top_w, perm_w, he, hg, ye, top_idx, perm_row, slot_of, grp_off, attn_ws, scan_ws, decay_ws,
                 hb, mb, yb, hgr, hgb, yeb};
  tc.release();
  release_row_buffers();
  for (void* p : dev)
    if (p) cudaFree(p);
  for (float* p : rope_cos)
    if (p) cudaFree(p);
  for (float* p : rope_sin)
    if (p) cudaFree(p);
}

void GxModel::reset_slot(qie_engine* e, int seq) {
  if (state) cudaMemsetAsync(state + (size_t)seq * slot_floats, 0, slot_floats * sizeof(float), e->stream);
}

cudaError_t GxModel::forward(qie_engine* e, int n, int n_seg, int n_out, int max_kv_len, float temperature, bool advance) {
  GxModel* m = this;
  cudaStream_t st = e->stream;
  const int W = m->width;
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
    if (cudaMalloc(&m->layer_dump, m->runs.size() * R * W * sizeof(float)) != cudaSuccess) return cudaErrorMemoryAllocation;
  // a norm step; `add` is what the sublayer before left to be added to the stream: projected mixer rows or the experts' rows
  enum Add { ADD_NONE, ADD_Y, ADD_YB, ADD_YE, ADD_YEB };
  Add add = ADD_NONE;
  int add_top = 0;
  auto step = [&](int rows) {
    GroupNormStep s;
    s.x = m->x, s.width = W, s.groups = 1, s.n = rows, s.eps = m->eps, s.w_off = 1.0f, s.embed = m->embed, s.embed_scale = m->embed_scale;
    if (add == ADD_Y) s.y1 = m->y;
    else if (add == ADD_YB) s.y1_bf = m->yb;
    else if (add == ADD_YE) s.mix.ye = m->ye;
    else if (add == ADD_YEB) s.ye_bf = m->yeb;
    if (add == ADD_YE || add == ADD_YEB) s.mix.slot_of = m->slot_of, s.mix.top = add_top;
    add = ADD_NONE;
    return s;
  };
  for (size_t ri = 0; ri < m->runs.size(); ++ri) {
    const GxRun& run = m->runs[ri];
    const GxLayer& L = m->layers[run.layer];
    const int ld = L.n_in, H = L.heads, d = L.dim, vd = L.vdim, nv = H * vd;
    const bool tc_in = tcfit(W, L.n_in, L.w_in), tc_o = tcfit(nv, W, L.wo);
    {  // x += outputs of the sublayer before (first run: the scaled embedding row); the embedding again; h = norm1(x)
      GroupNormStep s = step(n);
      if (ri == 0 || run.again) s.ids = e->ids_d, s.again = run.again;
      if (ri > 0 && m->dump_layers) s.dump = m->layer_dump + (ri - 1) * R * W;
      s.w_in = L.norm1;
      if (tc_in) s.h_bf = m->hb;
      else s.h = m->hn;
      FAM_TRY(KK_F32_NORM, launch_group_norm_step(s, st));
    }
    const bf16* pb = m->tc.cb;  // the input projection's result as bf16 rows
    if (tc_in) FAM_TRY(KK_F32_PROJ, m->tc.gemm_bf16(e, m->hb, L.w_in, W, L.n_in, m->tc.cb, n));
    else FAM_TRY(KK_F32_PROJ, proj(m->hn, W, L.w_in, W, L.n_in, m->p0, ld, n));
    // mixer -> rows mb (bf16, when the output projection takes them) or p1 (fp32)
    if (L.type == 0) {
      const int G = L.kv_heads;
      KvStoreArgs ks;
      ks.c.pool = m->kv_pool, ks.c.elt_bytes = m->f32 ? 4 : 2, ks.c.page_size = e->kv.page_size, ks.c.page_elems = m->page_elems;
      ks.c.layer_off = run.kv_off, ks.c.kw = G * d, ks.c.vw = G * vd, ks.c.n_pages = e->kv.n_pages;
      ks.unit_norm = 1, ks.norm_dim = d, ks.eps = m->eps, ks.q_heads = H;
      if (L.rope_id >= 0) ks.rope = RopeTable{m->rope_cos[L.rope_id], m->rope_sin[L.rope_id], L.rot.dims, 1};
      ks.pos = e->pos_d, ks.slot = e->slot_d, ks.block_table = e->block_table_d, ks.max_pages = e->max_pages_per_seq, ks.n = n;
      const float* q = m->p0 + L.o_q;
      int ldq = ld;
      bool bf_rows = false;
      if (tc_in) {  // straight from the projection's bf16 rows where the shape allows, else through fp32 rows
        ks.q_bf = pb + L.o_q, ks.k_bf = pb + L.o_k, ks.v_bf = pb + L.o_v, ks.ld_bf = ld, ks.q = m->p3, ks.ldq = H * d;
        bf_rows = kv_store_heads_fits(ks);
        if (bf_rows) {
          q = m->p3, ldq = H * d;
        } else {
          ks.q_bf = ks.k_bf = ks.v_bf = nullptr;
          FAM_TRY(KK_F32_PROJ, launch_rows_bf16_to_f32_ld(pb, ld, ld, m->p0, ld, n, st));
        }
      }
      if (!bf_rows) ks.k = m->p0 + L.o_k, ks.ldk = ld, ks.v = m->p0 + L.o_v, ks.ldv = ld, ks.q = m->p0 + L.o_q, ks.ldq = ld;
      FAM_TRY(KK_KV_STORE, launch_kv_store_rows(ks, st));  // rotated and normed keys, values -> cache rows; the queries alike
      GqaAttnArgs g;
      g.c = ks.c, g.q = q, g.ldq = ldq, g.out = m->p1, g.ldo = nv;
      if (tc_o) g.out_bf = m->mb, g.ldo_bf = nv;
      g.heads = H, g.kv_heads = G, g.dim = d, g.vdim = vd, g.scale = L.scale, g.chunk = L.chunk, g.eps = m->eps;
      g.pos = e->pos_d, g.slot = e->slot_d, g.block_table = e->block_table_d, g.max_pages = e->max_pages_per_seq, g.n = n, g.max_keys = max_kv_len;
      g.ws = m->attn_ws, g.ws_floats = m->attn_ws_floats, g.num_sms = e->num_sms;
      g.seg_start = segs, g.seg_slot = seg_sl, g.n_seg = n_seg;
      int nl = 0;
      FAM_TRY(KK_GQA_ATTN, launch_gqa_attention(g, st, &nl));
      e->launches += nl > 0 ? nl - 1 : 0;
    } else {
      LinearAttnArgs a;
      if (tc_in) a.q_bf = pb + L.o_q, a.k_bf = pb + L.o_k, a.v_bf = pb + L.o_v, a.g_bf = pb + L.o_g, a.gate.low_bf = pb + L.o_low, a.ld_bf = ld;
      else a.q = m->p0 + L.o_q, a.k = m->p0 + L.o_k, a.v = m->p0 + L.o_v, a.gate.low = m->p0 + L.o_low, a.ld = ld;
      a.q_scale = 1.0f / sqrtf((float)d);
      a.heads = H, a.dim = d, a.vdim = vd, a.eps = m->eps, a.norm_w = L.head_norm;
      a.gate.rank = L.rank, a.gate.a2 = L.a2, a.gate.bias = L.a2_b, a.gate.inv_tau = 1.0f / L.tau, a.gate.cum = m->decay_ws;
      a.out = m->p1, a.ldo = nv;
      a.state = m->state + run.state_off, a.slot_stride = m->slot_floats;
      a.seg_start = segs, a.seg_slot = seg_sl, a.n_seg = n_seg, a.n_rows = n;
      a.ws = m->scan_ws, a.ws_floats = m->scan_ws_floats;
      const bool fused = tc_o && linear_attention_norm_fits(a);
      if (fused) a.norm_gate = 1, a.out_bf = m->mb, a.ldo_bf = nv;
      int nl = 0;
      FAM_TRY(KK_LINEAR_ATTN, launch_linear_attention(a, st, &nl));
      e->launches += nl > 0 ? nl - 1 : 0;
      if (!fused) {
        NormGate g;
        g.v = m->p1, g.ldv = nv, g.width = nv, g.n = n, g.eps = m->eps, g.groups = H, g.act = 0, g.w = L.head_norm, g.w_shared = 1;
        if (tc_in) g.g_bf = pb + L.o_g, g.ldg_bf = ld;
        else g.g = m->p0 + L.o_g, g.ldg = ld;
        if (tc_o) g.out_bf = m->mb, g.ldo_bf = nv;
        else g.out = m->p1, g.ldo = nv;
        FAM_TRY(KK_NORM_GATE, launch_norm_gate(g, st));
      }
    }
    if (tc_o) FAM_TRY(KK_F32_PROJ, m->tc.gemm_bf16(e, m->mb, L.wo, nv, W, m->yb, n));
    else FAM_TRY(KK_F32_PROJ, proj(m->p1, nv, L.wo, nv, W, m->y, W, n));
    add = tc_o ? ADD_YB : ADD_Y;
    if (L.experts == 0) continue;
    // feed-forward: the router's weight scales the experts' input, which their two first maps let through
    const int E = L.experts, top = L.top, ff = L.ff;
    GroupedGemmBf16 eg, ed;
    bool tc_ex = false;
    if (!m->f32 && n * top > 16 * 16) {  // more rows than the GEMV serves
      eg.A = m->hb, eg.lda = W, eg.row_idx = m->perm_row, eg.grp_off = m->grp_off, eg.W = L.w_egu, eg.w_batch = (long)2 * ff * W;
      eg.N = 2 * ff, eg.K = W, eg.groups = E, eg.rows = n * top, eg.gated = 1, eg.out_bf = m->hgb, eg.ldo = ff, eg.row_w = m->perm_w, eg.a_rows = m->hgr;
      ed.A = m->hgb, ed.lda = ff, ed.grp_off = m->grp_off, ed.W = L.w_edown, ed.w_batch = (long)W * ff;
      ed.N = W, ed.K = ff, ed.groups = E, ed.rows = n * top, ed.out_bf = m->yeb, ed.ldo = W;
      tc_ex = grouped_gemm_bf16_fits(eg) && grouped_gemm_bf16_fits(ed);
    }
    {
      GroupNormStep s = step(n);
      s.w_in = L.norm2;
      if (tc_ex) s.h_bf = m->hb;
      else s.h = m->hn;
      s.route.w_router = L.w_router, s.route.experts = E, s.route.top = top, s.route.top_idx = m->top_idx, s.route.top_w = m->top_w;
      FAM_TRY(KK_F32_NORM, launch_group_norm_step(s, st));
    }
    FAM_TRY(KK_MOE_ROUTE, launch_moe_group(m->top_idx, n * top, top, E, m->grp_off, m->perm_row, m->slot_of, st, m->top_w, m->perm_w));
    if (tc_ex) {
      int nl = 0;
      FAM_TRY(KK_MOE_EXPERTS, launch_grouped_gemm_bf16(eg, st, e->num_sms, &nl));
      e->launches += nl > 0 ? nl - 1 : 0;
      FAM_TRY(KK_MOE_EXPERTS, launch_grouped_gemm_bf16(ed, st, e->num_sms));
    } else {
      GemmF32 g;  // [gate | up] of every assignment, rows grouped by expert and gathered from hn
      g.A = m->hn, g.lda = W, g.W = L.w_egu, g.ldw = W, g.w_batch = (long)2 * ff * W, g.C = m->he, g.ldc = 2 * ff;
      g.M = n * top, g.N = 2 * ff, g.K = W, g.batches = E, g.grp_off = m->grp_off, g.row_idx = m->perm_row, g.round_a = rnd;
      FAM_TRY(KK_MOE_EXPERTS, launch_gemm_f32(g, st));
      FAM_TRY(KK_GLU, launch_silu_glu(m->he, 2 * ff, m->hg, ff, ff, n * top, st, m->perm_w));
      GemmF32 g2;
      g2.A = m->hg, g2.lda = ff, g2.W = L.w_edown, g2.ldw = ff, g2.w_batch = (long)W * ff, g2.C = m->ye, g2.ldc = W;
      g2.M = n * top, g2.N = W, g2.K = ff, g2.batches = E, g2.grp_off = m->grp_off, g2.round_a = rnd;
      FAM_TRY(KK_MOE_EXPERTS, launch_gemm_f32(g2, st));
    }
    add = tc_ex ? ADD_YEB : ADD_YE, add_top = top;
  }
  if (m->dump_layers) {  // the last run's output meets the stream in every row, not only in the output rows
    GroupNormStep s = step(n);
    s.dump = m->layer_dump + (m->runs.size() - 1) * R * W;
    FAM_TRY(KK_F32_NORM, launch_group_norm_step(s, st));
  }
  if (n_out <= 0) return cudaSuccess;
  {
    GroupNormStep s = step(n_out);
    s.w_in = m->final_norm, s.h = m->xo, s.gather = outs;
    FAM_TRY(KK_F32_NORM, launch_group_norm_step(s, st));
  }
  {
    GemmF32 g;
    g.A = m->xo, g.lda = W, g.W = m->head, g.ldw = W, g.C = m->logits, g.ldc = m->vocab, g.M = n_out, g.N = m->vocab, g.K = W, g.round_a = rnd;
    FAM_TRY(KK_LM_HEAD, launch_gemm_f32(g, st));
    if (m->logit_scale != 1.0f || m->softcap > 0.f) FAM_TRY(KK_LM_HEAD, launch_softcap_f32(m->logits, (size_t)n_out * m->vocab, m->softcap, st, m->logit_scale));
  }
  return sample_rows(e, n_out, temperature, advance);
}

}  // namespace qie
