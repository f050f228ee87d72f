// Revitar: a decoder whose layers are listed one by one in config.json. Each layer is a sigmoid
// attention with a distance bias and a window (csrc/sigmoid_attention.cu), q and k normalised
// over their whole projections, and an optional layer of routed experts; norms sit on the
// sublayers' outputs only:
//
//   x = embed[token] * embedding.scale
//   x = x + m * norm1(attention(x));   x = x + m * norm2(experts(x))        m = residual_mult
//   logits = head . final_norm(x)
//
// config.json: architecture, vocab, width, embedding.scale, norm.eps, residual_mult and layers,
// a list of {type: "attention", mixer: {heads, kv_heads, dim, vdim, scale, softcap, mask.size},
// mlp: null or {kind: "moe", expert.ff, router.{experts, top}}}. Layers may differ in all of it.
// Tensors: embed, head, final.norm and, per layer, l<i>.{norm1, norm2}, l<i>.mix.{q, k, v, o,
// q.norm, k.norm, r1, r2, pb}, l<i>.mlp.router, l<i>.mlp.e<j>.{gate, up, down}.
//
// One or two rows (decoding) run on the row-streaming kernels, six launches a layer; more rows on
// the tile kernels, ten a layer. The residual stream, norms, scores, routing and all
// accumulation are f32 in both number formats.
#include <algorithm>

#include "dense_model.h"

namespace kanso {
namespace {

struct RevLayerSpec {
  uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, window = 0;
  float scale = 1.f, softcap = 0.f;
  uint32_t experts = 0, top = 0, ff = 0;  // experts 0: no feed-forward
};
struct RevConfig {
  uint32_t vocab = 0, width = 0;
  float embed_scale = 1.f, eps = 0.f, mult = 1.f;
  std::vector<RevLayerSpec> layers;
};

int32_t parse_config(kanso_cuda_ctx* ctx, const Json& j, RevConfig* c) {
  int32_t st;
  if ((st = need_size(ctx, j, "vocab", &c->vocab))) return st;
  if ((st = need_size(ctx, j, "width", &c->width))) return st;
  if ((st = need_float(ctx, j, "embedding.scale", &c->embed_scale))) return st;
  if ((st = need_float(ctx, j, "norm.eps", &c->eps))) return st;
  if ((st = need_float(ctx, j, "residual_mult", &c->mult))) return st;
  const Json* layers = j.find("layers");
  if (!layers || layers->kind != Json::ARR || layers->arr.empty())
    return fail(ctx, KANSO_ERR_CONFIG, "config.json: 'layers' is missing or empty");
  for (size_t i = 0; i < layers->arr.size(); ++i) {
    const Json& l = layers->arr[i];
    const Json *type = l.find("type"), *mix = l.find("mixer"), *mlp = l.find("mlp");
    if (!type || type->str != "attention")
      return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu has mixer type '%s' (known: "
                  "attention)", i, type ? type->str.c_str() : "");
    if (!mix || mix->kind != Json::OBJ)
      return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu has no 'mixer'", i);
    RevLayerSpec s;
    if ((st = need_size(ctx, *mix, "heads", &s.heads))) return st;
    if ((st = need_size(ctx, *mix, "kv_heads", &s.kv_heads))) return st;
    if ((st = need_size(ctx, *mix, "dim", &s.dim))) return st;
    if ((st = need_size(ctx, *mix, "vdim", &s.vdim))) return st;
    if ((st = need_float(ctx, *mix, "scale", &s.scale))) return st;
    const Json *cap = mix->find("softcap"), *mask = mix->find("mask");
    if (cap && !cap->is_null() && (st = need_float(ctx, *mix, "softcap", &s.softcap))) return st;
    if (mask && !mask->is_null() && (st = need_size(ctx, *mask, "size", &s.window))) return st;
    if (s.heads % s.kv_heads)
      return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu: %u heads over %u key/value heads",
                  i, s.heads, s.kv_heads);
    if (mlp && !mlp->is_null()) {
      const Json* kind = mlp->find("kind");
      if (kind && kind->str != "moe")
        return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu has feed-forward kind '%s' "
                    "(known: moe)", i, kind->str.c_str());
      if ((st = need_size(ctx, *mlp, "expert.ff", &s.ff))) return st;
      if ((st = need_size(ctx, *mlp, "router.experts", &s.experts))) return st;
      if ((st = need_size(ctx, *mlp, "router.top", &s.top))) return st;
      if (s.top > s.experts)
        return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu: top %u of %u experts", i,
                    s.top, s.experts);
    }
    c->layers.push_back(s);
  }
  return KANSO_OK;
}

uint32_t widest_window(const RevConfig& c) {
  uint32_t w = 0;
  for (const RevLayerSpec& s : c.layers) {
    if (!s.window) return 0;
    w = std::max(w, s.window);
  }
  return w;
}

struct RevLayer {
  DenseMat qkv, o, router, gate, up, down;
  float *norm1 = nullptr, *norm2 = nullptr, *q_norm = nullptr, *k_norm = nullptr;
  SigmoidAttn attn;
};

struct RevitarModel final : DenseModel {
  RevConfig cfg;
  std::vector<RevLayer> layers;
  DenseMat embed, head;
  float* final_norm = nullptr;
  // workspace of `ws_rows` rows
  int ws_parts = 1;
  float *x = nullptr, *x2 = nullptr, *qkv = nullptr, *oy = nullptr, *ao32 = nullptr,
        *rl = nullptr, *wgt = nullptr, *act32 = nullptr, *ye = nullptr;
  void *xe = nullptr, *q = nullptr, *ao = nullptr, *xs = nullptr, *act = nullptr;
  uint32_t *sel = nullptr, *slot = nullptr, *counts = nullptr, *offsets = nullptr;
  size_t counts_bytes = 0;

  const char* architecture() const override { return "Revitar"; }
  uint32_t vocab_size() const override { return cfg.vocab; }
  uint32_t num_layers() const override { return (uint32_t)cfg.layers.size(); }
  uint32_t max_window() const override { return widest_window(cfg); }
  std::vector<kanso_kv_layer> cache_layers() const override {
    std::vector<kanso_kv_layer> v;
    for (const RevLayerSpec& s : cfg.layers) v.push_back({s.kv_heads, s.dim, s.vdim, 0, 0, 0});
    return v;
  }

  int32_t load(const SafeTensors& st);

 private:
  int32_t ensure_ws(int64_t T);
  int32_t run(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev) override;
  int32_t run_rows(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev);
  int32_t run_tiles(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev);
  int32_t attend(kanso_cuda_kv* kv, size_t l, const DenseStep& s, const QkvSource& src, void* out,
                 bool out_f32, int64_t out_ld);
};

int32_t RevitarModel::load(const SafeTensors& st) {
  const bool f32 = compute == KANSO_COMPUTE_F32;
  const int64_t W = cfg.width, V = cfg.vocab;
  const StTensor* t = nullptr;
  int32_t e;
  if ((e = tensor(st, "embed", {V, W}, &t)) || (e = mat({t}, 1, W, f32, &embed))) return e;
  if ((e = tensor(st, "head", {V, W}, &t)) || (e = mat({t}, 1, W, f32, &head))) return e;
  if ((e = vec(st, "final.norm", W, &final_norm))) return e;
  layers.resize(cfg.layers.size());
  for (size_t i = 0; i < layers.size(); ++i) {
    const RevLayerSpec& s = cfg.layers[i];
    RevLayer& l = layers[i];
    const std::string p = "l" + std::to_string(i) + ".", mx = p + "mix.", ml = p + "mlp.";
    const int64_t nq = (int64_t)s.heads * s.dim, nk = (int64_t)s.kv_heads * s.dim,
                  nv = (int64_t)s.kv_heads * s.vdim, no = (int64_t)s.heads * s.vdim;
    const StTensor *tq, *tk, *tv;
    if ((e = tensor(st, mx + "q", {nq, W}, &tq)) || (e = tensor(st, mx + "k", {nk, W}, &tk)) ||
        (e = tensor(st, mx + "v", {nv, W}, &tv)) || (e = mat({tq, tk, tv}, 1, W, f32, &l.qkv)))
      return e;
    if ((e = tensor(st, mx + "o", {W, no}, &t)) || (e = mat({t}, 1, no, f32, &l.o))) return e;
    if ((e = vec(st, mx + "q.norm", nq, &l.q_norm)) || (e = vec(st, mx + "k.norm", nk, &l.k_norm)) ||
        (e = vec(st, p + "norm1", W, &l.norm1)))
      return e;
    std::vector<float> r1, r2, pb;
    if ((e = vec(st, mx + "r1", s.heads, nullptr, &r1)) ||
        (e = vec(st, mx + "r2", s.heads, nullptr, &r2)) ||
        (e = vec(st, mx + "pb", s.heads, nullptr, &pb)))
      return e;
    void* mem = nullptr;
    e = make_sigmoid_attn(ctx, s.heads, s.window, s.scale, s.softcap, r1.data(), r2.data(),
                          pb.data(), &l.attn, &mem);
    if (mem) owned.push_back(mem);
    if (e) return e;
    if (!s.experts) continue;
    if ((e = vec(st, p + "norm2", W, &l.norm2))) return e;
    if ((e = tensor(st, ml + "router", {s.experts, W}, &t)) || (e = mat({t}, 1, W, true, &l.router)))
      return e;
    std::vector<const StTensor*> g(s.experts), u(s.experts), d(s.experts);
    for (uint32_t x = 0; x < s.experts; ++x) {
      const std::string ex = ml + "e" + std::to_string(x) + ".";
      if ((e = tensor(st, ex + "gate", {s.ff, W}, &g[x])) ||
          (e = tensor(st, ex + "up", {s.ff, W}, &u[x])) ||
          (e = tensor(st, ex + "down", {W, s.ff}, &d[x])))
        return e;
    }
    if ((e = mat(g, s.experts, W, f32, &l.gate)) || (e = mat(u, s.experts, W, f32, &l.up)) ||
        (e = mat(d, s.experts, s.ff, f32, &l.down)))
      return e;
  }
  return KANSO_OK;
}

int32_t RevitarModel::ensure_ws(int64_t T) {
  if (T <= ws_rows) return KANSO_OK;
  ws_parts = T <= 512 ? 4 : 1;
  int64_t n_qkv = 0, n_q = 0, n_o = 0, ne = 0, nt = 0, nact = 0, nact32 = 0;
  for (const RevLayerSpec& s : cfg.layers) {
    n_qkv = std::max(n_qkv, (int64_t)s.heads * s.dim + (int64_t)s.kv_heads * (s.dim + s.vdim));
    n_q = std::max(n_q, (int64_t)s.heads * round_up8(s.dim));
    n_o = std::max(n_o, (int64_t)round_up8((int64_t)s.heads * s.vdim));
    ne = std::max(ne, (int64_t)s.experts);
    nt = std::max(nt, (int64_t)s.top);
    nact = std::max(nact, (int64_t)s.top * round_up8(s.ff));
    nact32 = nact;
  }
  const int64_t W = cfg.width, WL = round_up8(W);
  const size_t es = elem();
  counts_bytes = cfg.layers.size() * (size_t)ne * 4;
  return make_ws(T,
              {{(void**)&x, (size_t)(T * W) * 4},
               {(void**)&x2, (size_t)(T * W) * 4},
               {(void**)&qkv, (size_t)(ws_parts * T * n_qkv) * 4},
               {(void**)&oy, (size_t)(ws_parts * T * W) * 4},
               {(void**)&ao32, (size_t)(std::min<int64_t>(T, GEMV_MAX_T) * n_o) * 4},
               {(void**)&act32, (size_t)(std::min<int64_t>(T, GEMV_MAX_T) * nact32) * 4},
               {(void**)&rl, (size_t)(std::min<int64_t>(T, GEMV_MAX_T) * ne) * 4},
               {(void**)&wgt, (size_t)(T * nt) * 4},
               {(void**)&ye, (size_t)(T * nt * W) * 4},
               {&xe, (size_t)(T * WL) * es},
               {&q, (size_t)(T * n_q) * es},
               {&ao, (size_t)(T * n_o) * es},
               {&xs, (size_t)(T * nt * WL) * es},
               {&act, (size_t)(T * nact) * es},
               {(void**)&sel, (size_t)(T * nt) * 4},
               {(void**)&slot, (size_t)(T * nt) * 4},
               {(void**)&counts, counts_bytes},
               {(void**)&offsets, (size_t)(ne + 1) * 4}});
}

// The attention of layer l from its projections: stores k and v and leaves the heads' outputs.
int32_t RevitarModel::attend(kanso_cuda_kv* kv, size_t l, const DenseStep& s, const QkvSource& src,
                             void* out, bool out_f32, int64_t out_ld) {
  const RevLayer& ly = layers[l];
  const KvDenseLayer& pool = kv->dense[l];
  if (s.one_each)
    return launch_sigmoid_attn_rows(ctx, compute, ly.attn, pool, nullptr, &src, s.map, s.max_keys,
                                    out, out_f32, out_ld, s.T);
  int32_t st = launch_qk_norm_store(ctx, compute, src, pool, ly.attn.heads, s.map, q, s.T);
  if (st) return st;
  if (s.use_tiles && compute == KANSO_COMPUTE_BF16) {
    bool handled = false;
    st = launch_sigmoid_attn_prefill(ctx, ly.attn, pool, q, s.T, s.map, s.tiles128, s.n_tiles128,
                                     out, out_f32, out_ld, &handled);
    if (st || handled) return st;
    st = launch_sigmoid_attn_tiles(ctx, ly.attn, pool, q, s.map, s.tiles64, s.n_tiles64, out,
                                   out_f32, out_ld, &handled);
    if (st || handled) return st;
  }
  return launch_sigmoid_attn_rows(ctx, compute, ly.attn, pool, q, nullptr, s.map, s.max_keys, out,
                                  out_f32, out_ld, s.T);
}

int32_t RevitarModel::run(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev) {
  int32_t st = ensure_ws(s.T);
  if (st) return st;
  // the row-streaming down product keeps a row's chosen experts' activations in shared memory
  bool stream = s.T <= GEMV_MAX_T;
  for (const RevLayerSpec& l : cfg.layers)
    stream = stream && (int64_t)l.top * round_up8(l.ff) <= GEMV_MAX_COLS;
  return stream ? run_rows(kv, s, logits_dev) : run_tiles(kv, s, logits_dev);
}

// One or two rows: six launches per layer. The residual step of a sublayer runs in front of the
// product that reads its result: the router's for the attention, the next layer's qkv for the
// experts.
int32_t RevitarModel::run_rows(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev) {
  const int T = (int)s.T;
  const int64_t W = cfg.width;
  int32_t st;
  if ((st = launch_embed_scaled(ctx, compute, embed.w, embed.ld, s.tokens, cfg.vocab,
                                cfg.embed_scale, x, W, nullptr, T)))
    return st;
  float *cur = x, *other = x2;
  const float *y = nullptr, *y_norm = nullptr;  // a sublayer's output that is not yet added
  // With many rows every CTA repeating the residual step costs more than a launch of it.
  const bool fold = (int64_t)T * W <= 16384;
  auto source = [&](GemvSource* g) -> int32_t {
    *g = GemvSource();
    g->eps = cfg.eps;
    g->mult = cfg.mult;
    if (y && !fold) {
      ResidualSource r;
      r.y = y;
      const int32_t e = launch_residual_norm(ctx, compute, cur, W, r, y_norm, cfg.eps, cfg.mult,
                                             Residual::kAdd, nullptr, 0, T);
      if (e) return e;
      y = nullptr;
    }
    g->x = cur;
    if (y) {
      g->x_out = other;
      g->y = y;
      g->norm_w = y_norm;
      std::swap(cur, other);
      y = nullptr;
    }
    return KANSO_OK;
  };
  GemvSource g;
  for (size_t l = 0; l < layers.size(); ++l) {
    const RevLayer& ly = layers[l];
    const RevLayerSpec& sp = cfg.layers[l];
    if ((st = source(&g))) return st;
    if ((st = launch_gemv(ctx, compute, ly.qkv, g, qkv, ly.qkv.rows, T))) return st;
    QkvSource src;
    src.qkv = qkv;
    src.q_norm = ly.q_norm;
    src.k_norm = ly.k_norm;
    src.eps = cfg.eps;
    if ((st = attend(kv, l, s, src, ao32, true, ly.o.cols))) return st;
    g = GemvSource();
    g.x = ao32;
    if ((st = launch_gemv(ctx, compute, ly.o, g, oy, W, T))) return st;
    y = oy;
    y_norm = ly.norm1;
    if (!sp.experts) continue;
    if ((st = source(&g))) return st;
    if ((st = launch_gemv(ctx, KANSO_COMPUTE_F32, ly.router, g, rl, sp.experts, T))) return st;
    if ((st = launch_gemv_gate_up(ctx, compute, &ly.gate, ly.up, cur, rl, sp.experts, sp.top,
                                  RouteWeights::kShares, act32, sel, T)))
      return st;
    if ((st = launch_gemv_down(ctx, compute, ly.down, act32, sel, sp.top, ye, T))) return st;
    y = ye;
    y_norm = ly.norm2;
  }
  if (!s.n_want) return KANSO_OK;
  if ((st = source(&g))) return st;
  g.x_out = nullptr;
  g.final_w = final_norm;
  g.row_index = s.want;
  return launch_gemv(ctx, compute, head, g, logits_dev, cfg.vocab, (int)s.n_want);
}

int32_t RevitarModel::run_tiles(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev) {
  const int64_t T = s.T, W = cfg.width, WL = round_up8(W);
  int32_t st;
  int splits = 1;
  const int max_splits = T <= 512 ? ws_parts : 1;
  GemmRows rows;
  rows.T = T;
  if ((st = launch_embed_scaled(ctx, compute, embed.w, embed.ld, s.tokens, cfg.vocab,
                                cfg.embed_scale, x, W, xe, T)))
    return st;
  if (counts_bytes)
    KANSO_CUDA_TRY(ctx, cudaMemsetAsync(counts, 0, counts_bytes, ctx->stream), "expert counts");
  const size_t count_step = counts_bytes / 4 / layers.size();
  for (size_t l = 0; l < layers.size(); ++l) {
    const RevLayer& ly = layers[l];
    const RevLayerSpec& sp = cfg.layers[l];
    QkvSource src;
    src.qkv = qkv;
    src.part_stride = T * ly.qkv.rows;
    src.q_norm = ly.q_norm;
    src.k_norm = ly.k_norm;
    src.eps = cfg.eps;
    if ((st = launch_gemm(ctx, compute, ly.qkv, xe, qkv, ly.qkv.rows, rows, max_splits, &src.parts,
                          src.part_stride)))
      return st;
    if ((st = attend(kv, l, s, src, ao, false, ly.o.ld))) return st;
    if ((st = launch_gemm(ctx, compute, ly.o, ao, oy, W, rows, max_splits, &splits, T * W)))
      return st;
    ResidualSource r;
    r.y = oy;
    r.parts = splits;
    r.part_stride = T * W;
    if ((st = launch_residual_norm(ctx, compute, x, W, r, ly.norm1, cfg.eps, cfg.mult,
                                   Residual::kAdd, xe, WL, T)))
      return st;
    if (!sp.experts) continue;
    uint32_t* cnt = counts + l * count_step;
    if ((st = launch_route(ctx, x, W, ly.router, nullptr, sp.top, RouteWeights::kShares, sel, wgt,
                           cnt, slot, T))) return st;
    if ((st = launch_expert_gather(ctx, compute, cnt, sp.experts, sp.top, sel, slot, offsets, xe,
                                   WL, xs, T)))
      return st;
    GemmRows er;
    er.T = T * sp.top;
    er.offsets = offsets;
    er.groups = (int)sp.experts;
    if ((st = launch_gemm_gate_up(ctx, compute, ly.gate, ly.up, xs, act, ly.down.ld, er))) return st;
    if ((st = launch_gemm(ctx, compute, ly.down, act, ye, W, er, 1, &splits, 0))) return st;
    r = ResidualSource();
    r.y = ye;
    r.slot = slot;
    r.weight = wgt;
    r.top = (int)sp.top;
    if ((st = launch_residual_norm(ctx, compute, x, W, r, ly.norm2, cfg.eps, cfg.mult,
                                   Residual::kAdd, xe, WL, T)))
      return st;
  }
  return logits_of_rows(head, final_norm, cfg.eps, x, xe, s, logits_dev);
}

int32_t describe(kanso_cuda_ctx* ctx, const Json& config, std::string* summary) {
  RevConfig c;
  const int32_t st = parse_config(ctx, config, &c);
  if (st) return st;
  uint64_t kv = 0;
  for (const RevLayerSpec& s : c.layers)
    kv += (uint64_t)s.kv_heads * (round_up8(s.dim) + round_up8(s.vdim)) * 2;
  *summary = "{\"architecture\": \"Revitar\", \"layers\": " + std::to_string(c.layers.size()) +
             ", \"vocab\": " + std::to_string(c.vocab) + ", \"width\": " + std::to_string(c.width) +
             ", \"max_window\": " + std::to_string(widest_window(c)) +
             ", \"kv_bytes_per_token_bf16\": " + std::to_string(kv) + "}";
  return KANSO_OK;
}

int32_t load(kanso_cuda_ctx* ctx, const Json& config, const std::string& dir, int32_t compute,
             kanso_cuda_model** out) {
  std::unique_ptr<RevitarModel> m(new RevitarModel);
  m->ctx = ctx;
  m->compute = compute;
  int32_t st = parse_config(ctx, config, &m->cfg);
  SafeTensors file;
  if (!st) st = file.open(ctx, dir + "/model.safetensors");
  if (!st) st = m->load(file);
  if (st) return st;
  *out = m.release();
  return KANSO_OK;
}

const ModelRegistrar registered({"Revitar", describe, load});

}  // namespace
}  // namespace kanso
