// Migurax: a decoder whose layers are listed one by one in config.json. A layer is one of two
// mixers and an optional feed-forward, with the norm after each sum:
//
//   x = embed[token]
//   x = norm1(alpha * x + mixer(x));   x = norm2(alpha * x + ff(x))
//   logits = head . final_norm(x)
//
// Mixers: latent attention with a sink (csrc/latent_attention.cu, csrc/softmax_prefill.cu), which
// caches a normed latent and one rotated key part per token, and a matrix memory with exponential
// gates (csrc/mlstm.cu), which keeps a state per sequence. Feed-forwards: dense with biases, or routed
// experts weighted by the softmax over the chosen ones; both W_down relu(W_up h)^2.
//
// config.json: architecture, vocab, width, norm.eps, postln_alpha and layers, a list of {type, mixer,
// mlp}; type "latent_attention" with mixer {heads, dim, rot_dim, vdim, kv_rank, q_rank, scale,
// rot.{base, dims}}, type "mlstm" with mixer {heads, dim, vdim, gate_cap}; mlp null, {kind: "dense",
// ff} or {kind: "moe", expert.ff, router.{experts, top}}. Layers may differ in all of it.
// Tensors: embed, head, final.norm and, per layer, l<i>.{norm1, norm2}, l<i>.mix.{dq, dq.norm, uq,
// dkv, dkv.norm, uk, uv, sink, o} or l<i>.mix.{q, k, v, g, o, norm, i, i.b, f, f.b}, l<i>.mlp.{up,
// up.b, down, down.b} or l<i>.mlp.{router, router.b, e<j>.up, e<j>.down}.
//
// One or two sequences with a token each run on the row-streaming kernels, other steps on the tile
// kernels. The residual stream, norms, angles, scores, gates, states, routing and all accumulation
// are f32 in both number formats.
//
// A latent layer has two forms of its attention. Decoding and short portions work on the cached
// latents themselves: the queries go through the transposed key projection, the weighted latents
// through the value projection. Longer portions expand the latents of all visible tokens to keys
// and values first, which costs less arithmetic per pair of tokens.
#include <algorithm>

#include "dense_model.h"

namespace kanso {
namespace {

struct MigLayerSpec {
  bool latent = false;
  uint32_t heads = 0, dim = 0, vdim = 0;
  uint32_t rot = 0, kv_rank = 0, q_rank = 0;  // latent attention
  float scale = 1.f, cap = 1.f;
  double rot_base = 1.0;
  uint32_t ff = 0, experts = 0, top = 0;  // ff 0: no feed-forward; experts 0: dense
  int64_t down_rows() const { return (int64_t)q_rank + kv_rank + rot; }
  int64_t q_cols() const { return (int64_t)heads * (dim + rot); }
  int64_t out_cols() const { return (int64_t)heads * vdim; }
  int64_t memory_rows() const { return (int64_t)heads * (2 * dim + 2 * vdim + 2); }
  // keys and values of a token, heads padded to 8 columns
  int64_t kv_cols() const { return (int64_t)heads * (round_up8(dim) + round_up8(vdim)); }
};
struct MigConfig {
  uint32_t vocab = 0, width = 0;
  float eps = 0.f, alpha = 1.f;
  std::vector<MigLayerSpec> layers;
};

int32_t parse_mlp(kanso_cuda_ctx* ctx, const Json& mlp, size_t i, MigLayerSpec* s) {
  const Json* kind = mlp.find("kind");
  const std::string k = kind ? kind->str : "";
  if (k == "dense") return need_size(ctx, mlp, "ff", &s->ff);
  if (k != "moe")
    return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu has feed-forward kind '%s' (known: "
                "dense, moe)", i, k.c_str());
  int32_t st;
  if ((st = need_size(ctx, mlp, "expert.ff", &s->ff))) return st;
  if ((st = need_size(ctx, mlp, "router.experts", &s->experts))) return st;
  if ((st = need_size(ctx, mlp, "router.top", &s->top))) return st;
  if (s->top > s->experts)
    return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu: top %u of %u experts", i, s->top,
                s->experts);
  return KANSO_OK;
}

int32_t parse_config(kanso_cuda_ctx* ctx, const Json& j, MigConfig* c) {
  int32_t st;
  if ((st = need_size(ctx, j, "vocab", &c->vocab))) return st;
  if ((st = need_size(ctx, j, "width", &c->width))) return st;
  if ((st = need_float(ctx, j, "norm.eps", &c->eps))) return st;
  if ((st = need_float(ctx, j, "postln_alpha", &c->alpha))) return st;
  const Json* layers = j.find("layers");
  if (!layers || layers->kind != Json::ARR || layers->arr.empty())
    return fail(ctx, KANSO_ERR_CONFIG, "config.json: 'layers' is missing or empty");
  for (size_t i = 0; i < layers->arr.size(); ++i) {
    const Json& l = layers->arr[i];
    const Json *type = l.find("type"), *mix = l.find("mixer"), *mlp = l.find("mlp");
    const std::string name = type ? type->str : "";
    if (name != "latent_attention" && name != "mlstm")
      return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu has mixer type '%s' (known: "
                  "latent_attention, mlstm)", i, name.c_str());
    if (!mix || mix->kind != Json::OBJ)
      return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu has no 'mixer'", i);
    MigLayerSpec s;
    s.latent = name == "latent_attention";
    if ((st = need_size(ctx, *mix, "heads", &s.heads))) return st;
    if ((st = need_size(ctx, *mix, "dim", &s.dim))) return st;
    if ((st = need_size(ctx, *mix, "vdim", &s.vdim))) return st;
    if (s.latent) {
      uint32_t dims = 0;
      if ((st = need_size(ctx, *mix, "rot_dim", &s.rot))) return st;
      if ((st = need_size(ctx, *mix, "kv_rank", &s.kv_rank))) return st;
      if ((st = need_size(ctx, *mix, "q_rank", &s.q_rank))) return st;
      if ((st = need_float(ctx, *mix, "scale", &s.scale))) return st;
      if ((st = need_num(ctx, *mix, "rot.base", &s.rot_base))) return st;
      if ((st = need_size(ctx, *mix, "rot.dims", &dims))) return st;
      if (dims != s.rot || dims % 2)
        return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu rotates %u of %u columns", i,
                    dims, s.rot);
      if (!(s.rot_base > 0))
        return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu: 'rot.base' is not positive", i);
    } else {
      if ((st = need_float(ctx, *mix, "gate_cap", &s.cap))) return st;
      if (!(s.cap > 0))
        return fail(ctx, KANSO_ERR_CONFIG, "config.json: layer %zu: 'gate_cap' is not positive", i);
    }
    if (mlp && !mlp->is_null() && (st = parse_mlp(ctx, *mlp, i, &s))) return st;
    c->layers.push_back(s);
  }
  return KANSO_OK;
}

struct MigLayer {
  float *norm1 = nullptr, *norm2 = nullptr;
  DenseMat o;
  // latent attention
  DenseMat down, uq, uk_t, uv, ukv;  // uk_t, uv: a group per head; ukv: keys and values of all heads
  float *dq_norm = nullptr, *dkv_norm = nullptr;
  LatentAttn attn;
  // matrix memory
  DenseMat in;
  float* head_norm = nullptr;
  MlstmArgs memory;
  // feed-forward
  DenseMat up, ff_down, router;
  float *up_b = nullptr, *down_b = nullptr, *router_b = nullptr;
};

// Keys and values of one layer's prompts beyond this are not expanded.
constexpr int64_t EXPAND_MAX_BYTES = 16ll << 30;

struct MiguraxModel final : DenseModel {
  MigConfig cfg;
  std::vector<MigLayer> layers;
  DenseMat embed, head;
  float* final_norm = nullptr;
  // workspace of `ws_rows` rows
  int ws_parts = 1;
  float *x = nullptr, *x2 = nullptr, *y = nullptr, *q = nullptr, *q_lat = nullptr,
        *o_lat32 = nullptr, *mix32 = nullptr, *act32 = nullptr, *oy = nullptr, *ye = nullptr,
        *rl = nullptr, *wgt = nullptr;
  void *xe = nullptr, *cq = nullptr, *qh = nullptr, *q_rot = nullptr, *o_lat = nullptr, *ao = nullptr,
       *xs = nullptr, *act = nullptr, *chunk_mem = nullptr;
  uint32_t *sel = nullptr, *slot = nullptr, *counts = nullptr, *offsets = nullptr;
  size_t counts_bytes = 0;
  // expanded keys and values of the prompts of a step, grown on demand
  uint8_t* expand_mem = nullptr;
  size_t expand_bytes = 0;

  ~MiguraxModel() override {
    if (expand_mem) cudaFree(expand_mem);
  }
  const char* architecture() const override { return "Migurax"; }
  uint32_t vocab_size() const override { return cfg.vocab; }
  uint32_t num_layers() const override { return (uint32_t)cfg.layers.size(); }
  bool has_state() const override {
    for (const MigLayerSpec& s : cfg.layers)
      if (!s.latent) return true;
    return false;
  }
  std::vector<kanso_kv_layer> cache_layers() const override {
    std::vector<kanso_kv_layer> v;
    for (const MigLayerSpec& s : cfg.layers)
      v.push_back(s.latent ? kanso_kv_layer{1, s.kv_rank + s.rot, 0, 0, 0, 0}
                           : kanso_kv_layer{0, 0, 0, s.heads, s.dim, s.vdim});
    return v;
  }

  int32_t load(const SafeTensors& st);

 private:
  int32_t load_latent(const SafeTensors& st, const std::string& p, const MigLayerSpec& s,
                      MigLayer* l);
  int32_t load_memory(const SafeTensors& st, const std::string& p, const MigLayerSpec& s,
                      MigLayer* l);
  int32_t load_mlp(const SafeTensors& st, const std::string& p, const MigLayerSpec& s, MigLayer* l);
  int32_t ensure_ws(int64_t T);
  int32_t run(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev) override;
  int32_t run_rows(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev);
  int32_t run_tiles(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev);
  LatentStore store_of(kanso_cuda_kv* kv, size_t l, const DenseStep& s, int parts) const;
  MlstmArgs memory_of(kanso_cuda_kv* kv, size_t l, const DenseStep& s, int parts) const;
  int32_t latent_tiles(kanso_cuda_kv* kv, size_t l, const DenseStep& s);
  int32_t latent_short(kanso_cuda_kv* kv, size_t l, const DenseStep& s, const LatentQuery& lq,
                       const uint32_t* rows, int64_t n);
  int32_t latent_long(kanso_cuda_kv* kv, size_t l, const DenseStep& s, const LatentQuery& lq,
                      SoftmaxPrefill* p);
  int32_t memory_tiles(kanso_cuda_kv* kv, size_t l, const DenseStep& s);
};

int32_t MiguraxModel::load_latent(const SafeTensors& st, const std::string& p,
                                  const MigLayerSpec& s, MigLayer* l) {
  const bool f32 = compute == KANSO_COMPUTE_F32;
  const int64_t W = cfg.width, H = s.heads, D = s.dim, V = s.vdim, R = s.kv_rank;
  const StTensor *a = nullptr, *b = nullptr;
  int32_t e;
  if ((e = tensor(st, p + "dq", {s.q_rank, W}, &a)) ||
      (e = tensor(st, p + "dkv", {R + s.rot, W}, &b)) || (e = mat({a, b}, 1, W, f32, &l->down)) ||
      (e = tensor(st, p + "uq", {s.q_cols(), s.q_rank}, &a)) ||
      (e = mat({a}, 1, s.q_rank, f32, &l->uq)) || (e = tensor(st, p + "uk", {H * D, R}, &a)) ||
      (e = tensor(st, p + "uv", {H * V, R}, &b)) || (e = mat_transposed(a, D, R, f32, &l->uk_t)) ||
      (e = mat({b}, H, R, f32, &l->uv)))
    return e;
  if (!f32) {
    const int64_t D8 = round_up8(D), V8 = round_up8(V);
    if ((e = mat_rows({a, b}, s.kv_cols(), 1, R, false, [=](int64_t r) -> int64_t {
          const bool key = r < H * D8;
          const int64_t i = key ? r : r - H * D8, ld = key ? D8 : V8, n = key ? D : V;
          return i % ld < n ? (key ? 0 : H * D) + i / ld * n + i % ld : -1;
        }, &l->ukv)))
      return e;
  }
  float* sink = nullptr;
  void* freq = nullptr;
  const std::vector<double> f = rope_frequencies(s.rot, s.rot_base);
  if ((e = vec(st, p + "dq.norm", s.q_rank, &l->dq_norm)) ||
      (e = vec(st, p + "dkv.norm", R, &l->dkv_norm)) || (e = vec(st, p + "sink", H, &sink)) ||
      (e = upload(f.data(), f.size() * sizeof(double), &freq)))
    return e;
  l->attn.heads = s.heads;
  l->attn.dim = s.dim;
  l->attn.rot = s.rot;
  l->attn.vdim = s.vdim;
  l->attn.rank = s.kv_rank;
  l->attn.scale = s.scale;
  l->attn.sink = sink;
  l->attn.freq = static_cast<const double*>(freq);
  return KANSO_OK;
}

int32_t MiguraxModel::load_memory(const SafeTensors& st, const std::string& p,
                                  const MigLayerSpec& s, MigLayer* l) {
  const bool f32 = compute == KANSO_COMPUTE_F32;
  const int64_t W = cfg.width, H = s.heads;
  const StTensor* t[6];
  const struct {
    const char* name;
    int64_t rows;
  } parts[6] = {{"q", H * s.dim}, {"k", H * s.dim}, {"v", H * s.vdim},
                {"g", H * s.vdim}, {"i", H}, {"f", H}};
  int32_t e;
  for (int i = 0; i < 6; ++i)
    if ((e = tensor(st, p + parts[i].name, {parts[i].rows, W}, &t[i]))) return e;
  float *ib = nullptr, *fb = nullptr;
  if ((e = mat({t[0], t[1], t[2], t[3], t[4], t[5]}, 1, W, f32, &l->in)) ||
      (e = vec(st, p + "i.b", H, &ib)) || (e = vec(st, p + "f.b", H, &fb)) ||
      (e = vec(st, p + "norm", s.out_cols(), &l->head_norm)))
    return e;
  l->memory.heads = s.heads;
  l->memory.dim = s.dim;
  l->memory.vdim = s.vdim;
  l->memory.cap = s.cap;
  l->memory.i_bias = ib;
  l->memory.f_bias = fb;
  return KANSO_OK;
}

int32_t MiguraxModel::load_mlp(const SafeTensors& st, const std::string& p, const MigLayerSpec& s,
                               MigLayer* l) {
  const bool f32 = compute == KANSO_COMPUTE_F32;
  const int64_t W = cfg.width;
  const StTensor *a = nullptr, *b = nullptr;
  int32_t e;
  if (!s.experts) {
    if ((e = tensor(st, p + "up", {s.ff, W}, &a)) || (e = mat({a}, 1, W, f32, &l->up)) ||
        (e = tensor(st, p + "down", {W, s.ff}, &b)) || (e = mat({b}, 1, s.ff, f32, &l->ff_down)) ||
        (e = vec(st, p + "up.b", s.ff, &l->up_b)))
      return e;
    return vec(st, p + "down.b", W, &l->down_b);
  }
  if ((e = tensor(st, p + "router", {s.experts, W}, &a)) || (e = mat({a}, 1, W, true, &l->router)) ||
      (e = vec(st, p + "router.b", s.experts, &l->router_b)))
    return e;
  std::vector<const StTensor*> u(s.experts), d(s.experts);
  for (uint32_t x = 0; x < s.experts; ++x) {
    const std::string ex = p + "e" + std::to_string(x) + ".";
    if ((e = tensor(st, ex + "up", {s.ff, W}, &u[x])) ||
        (e = tensor(st, ex + "down", {W, s.ff}, &d[x])))
      return e;
  }
  if ((e = mat(u, s.experts, W, f32, &l->up))) return e;
  return mat(d, s.experts, s.ff, f32, &l->ff_down);
}

int32_t MiguraxModel::load(const SafeTensors& st) {
  const bool f32 = compute == KANSO_COMPUTE_F32;
  const int64_t W = cfg.width, V = cfg.vocab;
  const StTensor* t = nullptr;
  int32_t e;
  if ((e = tensor(st, "embed", {V, W}, &t)) || (e = mat({t}, 1, W, f32, &embed))) return e;
  if ((e = tensor(st, "head", {V, W}, &t)) || (e = mat({t}, 1, W, f32, &head))) return e;
  if ((e = vec(st, "final.norm", W, &final_norm))) return e;
  layers.resize(cfg.layers.size());
  for (size_t i = 0; i < layers.size(); ++i) {
    const MigLayerSpec& s = cfg.layers[i];
    MigLayer& l = layers[i];
    const std::string p = "l" + std::to_string(i) + ".", mx = p + "mix.";
    if ((e = vec(st, p + "norm1", W, &l.norm1)) ||
        (e = s.latent ? load_latent(st, mx, s, &l) : load_memory(st, mx, s, &l)) ||
        (e = tensor(st, mx + "o", {W, s.out_cols()}, &t)) ||
        (e = mat({t}, 1, s.out_cols(), f32, &l.o)))
      return e;
    if (s.ff && ((e = vec(st, p + "norm2", W, &l.norm2)) || (e = load_mlp(st, p + "mlp.", s, &l))))
      return e;
  }
  return KANSO_OK;
}

int32_t MiguraxModel::ensure_ws(int64_t T) {
  if (T <= ws_rows) return KANSO_OK;
  ws_parts = T <= 512 ? 4 : 1;
  int64_t ny = 0, nq = 0, n_cq = 0, n_qh = 0, n_qr = 0, n_lat = 0, n_o = 0, nact = 0, ne = 0, nt = 1;
  size_t chunk = 0;
  for (const MigLayerSpec& s : cfg.layers) {
    if (s.latent) {
      ny = std::max(ny, s.down_rows());
      nq = std::max(nq, s.q_cols());
      n_cq = std::max(n_cq, (int64_t)round_up8(s.q_rank));
      n_qh = std::max(n_qh, (int64_t)s.heads * round_up8(s.dim));
      n_qr = std::max(n_qr, (int64_t)s.heads * round_up8(s.rot));
      n_lat = std::max(n_lat, (int64_t)s.heads * round_up8(s.kv_rank));
    } else {
      ny = std::max(ny, s.memory_rows());
      chunk = std::max(chunk, mlstm_chunk_bytes(s.heads, s.dim, s.vdim, T));
    }
    n_o = std::max(n_o, (int64_t)round_up8(s.out_cols()));
    nact = std::max(nact, (int64_t)std::max(1u, s.top) * round_up8(s.ff));
    ne = std::max(ne, (int64_t)s.experts);
    nt = std::max(nt, (int64_t)s.top);
  }
  const int64_t W = cfg.width, WL = round_up8(W), few = std::min<int64_t>(T, GEMV_MAX_T);
  const size_t es = elem();
  counts_bytes = cfg.layers.size() * (size_t)ne * 4;
  return make_ws(T, {{(void**)&x, (size_t)(T * W) * 4},
                     {(void**)&x2, (size_t)(T * W) * 4},
                     {(void**)&y, (size_t)(ws_parts * T * ny) * 4},
                     {(void**)&q, (size_t)(ws_parts * T * nq) * 4},
                     {(void**)&q_lat, (size_t)(T * n_lat) * 4},
                     {(void**)&o_lat32, (size_t)(few * n_lat) * 4},
                     {(void**)&mix32, (size_t)(T * n_o) * 4},
                     {(void**)&act32, (size_t)(few * nact) * 4},
                     {(void**)&oy, (size_t)(ws_parts * T * W) * 4},
                     {(void**)&ye, (size_t)(T * nt * W) * 4},
                     {(void**)&rl, (size_t)(few * ne) * 4},
                     {(void**)&wgt, (size_t)(T * nt) * 4},
                     {&xe, (size_t)(T * WL) * es},
                     {&cq, (size_t)(T * n_cq) * es},
                     {&qh, (size_t)(2 * T * n_qh) * es},
                     {&q_rot, (size_t)(T * n_qr) * es},
                     {&o_lat, (size_t)(T * n_lat) * es},
                     {&ao, (size_t)(T * n_o) * es},
                     {&xs, (size_t)(T * nt * WL) * es},
                     {&act, (size_t)(T * nact) * es},
                     {&chunk_mem, compute == KANSO_COMPUTE_BF16 ? chunk : 0},
                     {(void**)&sel, (size_t)(T * nt) * 4},
                     {(void**)&slot, (size_t)(T * nt) * 4},
                     {(void**)&counts, counts_bytes},
                     {(void**)&offsets, (size_t)(ne + 1) * 4}});
}

int32_t MiguraxModel::run(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev) {
  int32_t st = ensure_ws(s.T);
  if (st) return st;
  // the row-streaming kernels keep their input rows in shared memory
  bool stream = s.one_each && s.T <= GEMV_MAX_T && cfg.width <= GEMV_MAX_COLS / 2;
  for (const MigLayerSpec& l : cfg.layers)
    stream = stream && (int64_t)std::max(1u, l.top) * round_up8(l.ff) <= GEMV_MAX_COLS &&
             l.out_cols() <= GEMV_MAX_COLS && l.q_rank <= GEMV_MAX_COLS;
  return stream ? run_rows(kv, s, logits_dev) : run_tiles(kv, s, logits_dev);
}

// The cache rows of layer l from the down projections in y.
LatentStore MiguraxModel::store_of(kanso_cuda_kv* kv, size_t l, const DenseStep& s,
                                   int parts) const {
  const MigLayerSpec& sp = cfg.layers[l];
  LatentStore t;
  t.a = layers[l].attn;
  t.down.d = y;
  t.down.parts = parts;
  t.down.ld = sp.down_rows();
  t.down.part_stride = s.T * sp.down_rows();
  t.down.q_rank = sp.q_rank;
  t.down.q_norm = layers[l].dq_norm;
  t.down.c_norm = layers[l].dkv_norm;
  t.down.eps = cfg.eps;
  t.kv = kv->dense[l];
  t.map = s.map;
  t.status = ctx->dev_status;
  return t;
}

// The matrix memory of layer l over the projections in y, its results in mix32.
MlstmArgs MiguraxModel::memory_of(kanso_cuda_kv* kv, size_t l, const DenseStep& s,
                                  int parts) const {
  MlstmArgs a = layers[l].memory;
  a.y = y;
  a.parts = parts;
  a.part_stride = s.T * cfg.layers[l].memory_rows();
  a.state = kv->state[l];
  a.positions = s.map.positions;
  a.portions = s.portions;
  a.slots = s.slots;
  a.out = mix32;
  return a;
}

// One token each of one or two sequences. The residual step of a sublayer runs in front of the
// product that reads its result.
int32_t MiguraxModel::run_rows(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev) {
  const int T = (int)s.T;
  const int64_t W = cfg.width;
  int32_t st;
  if ((st = launch_embed_scaled(ctx, compute, embed.w, embed.ld, s.tokens, cfg.vocab, 1.f, x, W,
                                nullptr, T)))
    return st;
  float *cur = x, *other = x2;
  const float *out = nullptr, *out_norm = nullptr;  // a sublayer's output that is not yet added
  // With many columns every CTA repeating the residual step costs more than a launch of it.
  const bool fold = (int64_t)T * W <= 16384;
  auto source = [&](GemvSource* g) -> int32_t {
    *g = GemvSource();
    g->eps = cfg.eps;
    g->mult = cfg.alpha;
    g->form = Residual::kAddNorm;
    if (out && !fold) {
      ResidualSource r;
      r.y = out;
      const int32_t e = launch_residual_norm(ctx, compute, cur, W, r, out_norm, cfg.eps, cfg.alpha,
                                             Residual::kAddNorm, nullptr, 0, T);
      if (e) return e;
      out = nullptr;
    }
    g->x = cur;
    if (out) {
      g->x_out = other;
      g->y = out;
      g->norm_w = out_norm;
      std::swap(cur, other);
      out = nullptr;
    }
    return KANSO_OK;
  };
  GemvSource g;
  for (size_t l = 0; l < layers.size(); ++l) {
    const MigLayer& ly = layers[l];
    const MigLayerSpec& sp = cfg.layers[l];
    if ((st = source(&g))) return st;
    if (sp.latent) {
      const int64_t H = sp.heads, R = sp.kv_rank, Q = sp.dim + sp.rot;
      if ((st = launch_gemv(ctx, compute, ly.down, g, y, ly.down.rows, T))) return st;
      const LatentStore store = store_of(kv, l, s, 1);
      g = GemvSource();
      g.x = y;
      g.x_ld = ly.down.rows;
      g.final_w = ly.dq_norm;
      g.eps = cfg.eps;
      if ((st = launch_gemv(ctx, compute, ly.uq, g, q, ly.uq.rows, T, GemvOut(), &store))) return st;
      g = GemvSource();
      g.x = q;
      g.x_ld = H * Q;
      g.x_group = Q;
      GemvOut go;
      go.group_step = R;
      if ((st = launch_gemv(ctx, compute, ly.uk_t, g, q_lat, H * R, T, go))) return st;
      LatentRows r;
      r.q_lat = q_lat;
      r.q_row = r.out_row = H * R;
      r.q_head = r.out_head = R;
      r.q.q = q;
      r.q.ld = H * Q;
      r.map = s.map;
      r.max_keys = s.max_keys;
      r.early = true;
      r.out = o_lat32;
      r.out_f32 = true;
      r.n = T;
      bool handled = false;
      if ((st = launch_latent_attn_rows(ctx, compute, ly.attn, kv->dense[l], r, 0, &handled)))
        return st;
      g = GemvSource();
      g.x = o_lat32;
      g.x_ld = H * R;
      g.x_group = R;
      go.group_step = sp.vdim;
      if ((st = launch_gemv(ctx, compute, ly.uv, g, mix32, ly.o.cols, T, go))) return st;
      g = GemvSource();
      g.x = mix32;
    } else {
      if ((st = launch_gemv(ctx, compute, ly.in, g, y, ly.in.rows, T))) return st;
      const MlstmArgs a = memory_of(kv, l, s, 1);
      if ((st = launch_mlstm_rows(ctx, a, T, 1))) return st;
      g = GemvSource();
      g.x = mix32;
      g.gate = y + (int64_t)sp.heads * (2 * sp.dim + sp.vdim);
      g.gate_ld = ly.in.rows;
      g.heads = (int)sp.heads;
      g.norm_w = ly.head_norm;
      g.eps = cfg.eps;
    }
    if ((st = launch_gemv(ctx, compute, ly.o, g, oy, W, T))) return st;
    out = oy;
    out_norm = ly.norm1;
    if (!sp.ff) continue;
    if ((st = source(&g))) return st;
    GemvOut go;
    if (sp.experts) {
      go.bias = ly.router_b;
      if ((st = launch_gemv(ctx, KANSO_COMPUTE_F32, ly.router, g, rl, sp.experts, T, go)) ||
          (st = launch_gemv_gate_up(ctx, compute, nullptr, ly.up, cur, rl, sp.experts, sp.top,
                                    RouteWeights::kChosenSoftmax, act32, sel, T)) ||
          (st = launch_gemv_down(ctx, compute, ly.ff_down, act32, sel, sp.top, ye, T)))
        return st;
      out = ye;
    } else {
      go.bias = ly.up_b;
      go.relu2 = true;
      if ((st = launch_gemv(ctx, compute, ly.up, g, act32, sp.ff, T, go))) return st;
      g = GemvSource();
      g.x = act32;
      go = GemvOut();
      go.bias = ly.down_b;
      if ((st = launch_gemv(ctx, compute, ly.ff_down, g, ye, W, T, go))) return st;
      out = ye;
    }
    out_norm = ly.norm2;
  }
  if (!s.n_want) return KANSO_OK;
  if ((st = source(&g))) return st;
  g.x_out = nullptr;
  g.final_w = final_norm;
  g.row_index = s.want;
  return launch_gemv(ctx, compute, head, g, logits_dev, cfg.vocab, (int)s.n_want);
}

// Attention on the latents for the listed rows; leaves the heads' outputs in ao.
int32_t MiguraxModel::latent_short(kanso_cuda_kv* kv, size_t l, const DenseStep& s,
                                   const LatentQuery& lq, const uint32_t* rows, int64_t n) {
  const MigLayer& ly = layers[l];
  const MigLayerSpec& sp = cfg.layers[l];
  const int64_t H = sp.heads, R = sp.kv_rank, RL = round_up8(R);
  int32_t st;
  int splits = 1;
  void* q_heads = static_cast<uint8_t*>(qh) + (size_t)s.T * H * round_up8(sp.dim) * elem();
  if ((st = launch_latent_q_heads(ctx, compute, ly.attn, lq, rows, n, q_heads))) return st;
  GemmRows hr;
  hr.T = H * n;
  hr.groups = (int)H;
  if ((st = launch_gemm(ctx, compute, ly.uk_t, q_heads, q_lat, R, hr, 1, &splits, 0))) return st;
  LatentRows r;
  r.q_lat = q_lat;
  r.q_row = R;
  r.q_head = n * R;
  r.q = lq;
  r.rows = rows;
  r.map = s.map;
  r.max_keys = s.max_keys;
  r.early = s.one_each;
  r.out = o_lat;
  r.out_row = RL;
  r.out_head = n * RL;
  r.n = n;
  bool handled = false;
  if ((st = launch_latent_attn_rows(ctx, compute, ly.attn, kv->dense[l], r, 0, &handled)))
    return st;
  GemmOut o;
  o.elem = true;
  o.group_step = sp.vdim;
  o.rows = rows;
  return launch_gemm(ctx, compute, ly.uv, o_lat, ao, ly.o.ld, hr, 1, &splits, 0, o);
}

// Attention of the long portions on expanded keys and values (bfloat16).
int32_t MiguraxModel::latent_long(kanso_cuda_kv* kv, size_t l, const DenseStep& s,
                                  const LatentQuery& lq, SoftmaxPrefill* p) {
  const MigLayer& ly = layers[l];
  const MigLayerSpec& sp = cfg.layers[l];
  const int64_t n = s.long_keys, N = sp.kv_cols(), RL = round_up8(sp.kv_rank),
                OL = round_up8(sp.rot);
  const size_t total = (size_t)n * (N + RL + OL) * 2 + 1024;
  if (total > expand_bytes) {
    cudaStreamSynchronize(ctx->stream);
    if (expand_mem) cudaFree(expand_mem);
    expand_mem = nullptr;
    expand_bytes = 0;
    KANSO_CUDA_TRY(ctx, cudaMalloc((void**)&expand_mem, total + total / 2), "expanded keys");
    expand_bytes = total + total / 2;
  }
  auto up = [](size_t b) { return (b + 255) & ~(size_t)255; };
  bf16* kvx = reinterpret_cast<bf16*>(expand_mem);
  bf16* c = reinterpret_cast<bf16*>(expand_mem + up((size_t)n * N * 2));
  bf16* rot = reinterpret_cast<bf16*>(expand_mem + up((size_t)n * N * 2) + up((size_t)n * RL * 2));
  int32_t st;
  int splits = 1;
  if ((st = launch_latent_q_rows(ctx, ly.attn, lq, s.map.positions, (bf16*)qh, (bf16*)q_rot, s.T)) ||
      (st = launch_latent_gather(ctx, ly.attn, kv->dense[l], s.map, s.key_runs, s.n_long, c, rot,
                                 n)))
    return st;
  GemmRows kr;
  kr.T = n;
  GemmOut o;
  o.elem = true;
  if ((st = launch_gemm(ctx, compute, ly.ukv, c, kvx, N, kr, 1, &splits, 0, o))) return st;
  p->q = (const bf16*)qh;
  p->q_rot = (const bf16*)q_rot;
  p->q_rows = s.T;
  p->k = kvx;
  p->v = kvx + (int64_t)sp.heads * round_up8(sp.dim);
  p->k_rot = rot;
  p->k_ld = p->v_ld = N;
  p->tiles = s.long_tiles;
  p->n_tiles = s.n_long_tiles;
  p->out = (bf16*)ao;
  p->out_ld = ly.o.ld;
  bool handled = false;
  if ((st = launch_softmax_prefill(ctx, *p, &handled))) return st;
  return handled ? KANSO_OK
                 : fail(ctx, KANSO_ERR_UNSUPPORTED, "prompt attention: %u heads of %u + %u and %u "
                                                    "columns", sp.heads, sp.dim, sp.rot, sp.vdim);
}

int32_t MiguraxModel::latent_tiles(kanso_cuda_kv* kv, size_t l, const DenseStep& s) {
  const MigLayer& ly = layers[l];
  const MigLayerSpec& sp = cfg.layers[l];
  const int64_t T = s.T;
  const int max_splits = T <= 512 ? ws_parts : 1;
  GemmRows rows;
  rows.T = T;
  int32_t st;
  int parts = 1;
  LatentQuery lq;
  lq.q = q;
  lq.ld = sp.q_cols();
  lq.part_stride = T * sp.q_cols();
  if ((st = launch_gemm(ctx, compute, ly.down, xe, y, ly.down.rows, rows, max_splits, &parts,
                        T * ly.down.rows)) ||
      (st = launch_latent_down(ctx, compute, store_of(kv, l, s, parts), cq, T)) ||
      (st = launch_gemm(ctx, compute, ly.uq, cq, q, sp.q_cols(), rows, max_splits, &lq.parts,
                        lq.part_stride)))
    return st;
  SoftmaxPrefill p;
  p.heads = sp.heads;
  p.dim = sp.dim;
  p.rot = sp.rot;
  p.vdim = sp.vdim;
  p.scale = sp.scale;
  p.sink = ly.attn.sink;
  p.keys = s.long_keys;
  if (!s.n_long || compute != KANSO_COMPUTE_BF16 || !softmax_prefill_fits(p) ||
      s.long_keys * sp.kv_cols() * 2 > EXPAND_MAX_BYTES)
    return latent_short(kv, l, s, lq, nullptr, T);
  if ((st = latent_long(kv, l, s, lq, &p))) return st;
  return s.n_short_rows ? latent_short(kv, l, s, lq, s.short_rows, s.n_short_rows) : KANSO_OK;
}

int32_t MiguraxModel::memory_tiles(kanso_cuda_kv* kv, size_t l, const DenseStep& s) {
  const MigLayer& ly = layers[l];
  GemmRows rows;
  rows.T = s.T;
  int32_t st;
  int parts = 1;
  if ((st = launch_gemm(ctx, compute, ly.in, xe, y, ly.in.rows, rows, s.T <= 512 ? ws_parts : 1,
                        &parts, s.T * ly.in.rows)))
    return st;
  const MlstmArgs a = memory_of(kv, l, s, parts);
  const bool chunks = s.n_long && compute == KANSO_COMPUTE_BF16 && mlstm_chunk_fits(a);
  const uint32_t by_row = chunks ? s.n_short : s.n_short + s.n_long;
  if (by_row &&
      (st = launch_mlstm_rows(ctx, a, by_row, chunks || !s.n_long ? s.max_short_rows : (uint32_t)s.T)))
    return st;
  if (chunks) {
    MlstmArgs b = a;
    b.portions = s.portions + s.n_short;
    if ((st = launch_mlstm_chunks(ctx, b, s.n_long, s.max_long_rows, chunk_mem, s.T))) return st;
  }
  return launch_head_norm_gate(ctx, compute, a, ly.head_norm, cfg.eps, ao, ly.o.ld, s.T);
}

int32_t MiguraxModel::run_tiles(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev) {
  const int64_t T = s.T, W = cfg.width, WL = round_up8(W);
  int32_t st;
  int splits = 1;
  const int max_splits = T <= 512 ? ws_parts : 1;
  GemmRows rows;
  rows.T = T;
  if ((st = launch_embed_scaled(ctx, compute, embed.w, embed.ld, s.tokens, cfg.vocab, 1.f, x, W, xe,
                                T)))
    return st;
  if (counts_bytes)
    KANSO_CUDA_TRY(ctx, cudaMemsetAsync(counts, 0, counts_bytes, ctx->stream), "expert counts");
  const size_t count_step = counts_bytes / 4 / layers.size();
  for (size_t l = 0; l < layers.size(); ++l) {
    const MigLayer& ly = layers[l];
    const MigLayerSpec& sp = cfg.layers[l];
    if ((st = sp.latent ? latent_tiles(kv, l, s) : memory_tiles(kv, l, s))) return st;
    if ((st = launch_gemm(ctx, compute, ly.o, ao, oy, W, rows, max_splits, &splits, T * W)))
      return st;
    ResidualSource r;
    r.y = oy;
    r.parts = splits;
    r.part_stride = T * W;
    if ((st = launch_residual_norm(ctx, compute, x, W, r, ly.norm1, cfg.eps, cfg.alpha,
                                   Residual::kAddNorm, xe, WL, T)))
      return st;
    if (!sp.ff) continue;
    GemmOut up_out;
    up_out.relu2 = up_out.elem = true;
    r = ResidualSource();
    if (sp.experts) {
      uint32_t* cnt = counts + l * count_step;
      GemmRows er;
      er.T = T * sp.top;
      er.offsets = offsets;
      er.groups = (int)sp.experts;
      if ((st = launch_route(ctx, x, W, ly.router, ly.router_b, sp.top,
                             RouteWeights::kChosenSoftmax, sel, wgt, cnt, slot, T)) ||
          (st = launch_expert_gather(ctx, compute, cnt, sp.experts, sp.top, sel, slot, offsets, xe,
                                     WL, xs, T)) ||
          (st = launch_gemm(ctx, compute, ly.up, xs, act, ly.ff_down.ld, er, 1, &splits, 0,
                            up_out)) ||
          (st = launch_gemm(ctx, compute, ly.ff_down, act, ye, W, er, 1, &splits, 0)))
        return st;
      r.y = ye;
      r.slot = slot;
      r.weight = wgt;
      r.top = (int)sp.top;
    } else {
      up_out.bias = ly.up_b;
      GemmOut down_out;
      down_out.bias = ly.down_b;
      if ((st = launch_gemm(ctx, compute, ly.up, xe, act, ly.ff_down.ld, rows, 1, &splits, 0,
                            up_out)) ||
          (st = launch_gemm(ctx, compute, ly.ff_down, act, oy, W, rows, max_splits, &splits, T * W,
                            down_out)))
        return st;
      r.y = oy;
      r.parts = splits;
      r.part_stride = T * W;
    }
    if ((st = launch_residual_norm(ctx, compute, x, W, r, ly.norm2, cfg.eps, cfg.alpha,
                                   Residual::kAddNorm, xe, WL, T)))
      return st;
  }
  return logits_of_rows(head, final_norm, cfg.eps, x, xe, s, logits_dev);
}

int32_t describe(kanso_cuda_ctx* ctx, const Json& config, std::string* summary) {
  MigConfig c;
  const int32_t st = parse_config(ctx, config, &c);
  if (st) return st;
  uint64_t kv = 0, state = 0;
  for (const MigLayerSpec& s : c.layers) {
    if (s.latent) {
      kv += (uint64_t)round_up8(s.kv_rank + s.rot) * 2;
    } else {
      KvStateLayer k;
      k.heads = s.heads;
      k.dim = s.dim;
      k.vdim = s.vdim;
      state += k.slot_floats() * 4;
    }
  }
  *summary = "{\"architecture\": \"Migurax\", \"layers\": " + std::to_string(c.layers.size()) +
             ", \"vocab\": " + std::to_string(c.vocab) + ", \"width\": " + std::to_string(c.width) +
             ", \"max_window\": 0, \"kv_bytes_per_token_bf16\": " + std::to_string(kv) +
             ", \"state_bytes_per_sequence\": " + std::to_string(state) + "}";
  return KANSO_OK;
}

int32_t load(kanso_cuda_ctx* ctx, const Json& config, const std::string& dir, int32_t compute,
             kanso_cuda_model** out) {
  std::unique_ptr<MiguraxModel> m(new MiguraxModel);
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

const ModelRegistrar registered({"Migurax", describe, load});

}  // namespace
}  // namespace kanso
