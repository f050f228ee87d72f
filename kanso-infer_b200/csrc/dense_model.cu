// The shared half of the unquantised model classes (dense_model.h).
#include "dense_model.h"

#include <algorithm>
#include <cstring>

namespace kanso {

int32_t need_num(kanso_cuda_ctx* ctx, const Json& j, const char* path, double* out) {
  const Json* at = &j;
  std::string rest(path);
  while (at && !rest.empty()) {
    const size_t dot = rest.find('.');
    at = at->find(rest.substr(0, dot).c_str());
    rest = dot == std::string::npos ? "" : rest.substr(dot + 1);
  }
  if (!at || at->kind != Json::NUM)
    return fail(ctx, KANSO_ERR_CONFIG, "config.json: '%s' is missing or not a number", path);
  *out = at->num;
  return KANSO_OK;
}
int32_t need_size(kanso_cuda_ctx* ctx, const Json& j, const char* path, uint32_t* out) {
  double v = 0;
  const int32_t st = need_num(ctx, j, path, &v);
  if (st) return st;
  if (v < 1 || v > 2147483647.0 || v != (double)(uint32_t)v)
    return fail(ctx, KANSO_ERR_CONFIG, "config.json: '%s' is not a positive whole number", path);
  *out = (uint32_t)v;
  return KANSO_OK;
}
int32_t need_float(kanso_cuda_ctx* ctx, const Json& j, const char* path, float* out) {
  double v = 0;
  const int32_t st = need_num(ctx, j, path, &v);
  *out = (float)v;
  return st;
}

static float st_value(const StTensor& t, int64_t i) {
  if (t.type == StType::BF16) {
    uint16_t h;
    std::memcpy(&h, t.data + 2 * i, 2);
    const uint32_t u = (uint32_t)h << 16;
    float f;
    std::memcpy(&f, &u, 4);
    return f;
  }
  float f;
  std::memcpy(&f, t.data + 4 * i, 4);
  return f;
}
static uint16_t bf16_bits(float f) {  // round to nearest, ties to even
  uint32_t u;
  std::memcpy(&u, &f, 4);
  if ((u & 0x7FFFFFFFu) > 0x7F800000u) return (uint16_t)((u >> 16) | 0x40u);
  return (uint16_t)((u + 0x7FFFu + ((u >> 16) & 1u)) >> 16);
}
static void put_value(uint8_t* dst, bool f32, float v) {
  if (f32) {
    std::memcpy(dst, &v, 4);
  } else {
    const uint16_t h = bf16_bits(v);
    std::memcpy(dst, &h, 2);
  }
}

int32_t DenseModel::tensor(const SafeTensors& st, const std::string& name,
                           std::vector<int64_t> shape, const StTensor** out) {
  const StTensor* t = st.find(name);
  if (!t) return fail(ctx, KANSO_ERR_CONFIG, "tensor '%s' is missing", name.c_str());
  if (t->shape != shape || t->type == StType::I32) {
    std::string want, got;
    for (int64_t d : shape) want += " " + std::to_string(d);
    for (int64_t d : t->shape) got += " " + std::to_string(d);
    return fail(ctx, KANSO_ERR_SHAPE, "tensor '%s' is [%s ], the configuration needs [%s ]",
                name.c_str(), got.c_str(), want.c_str());
  }
  *out = t;
  return KANSO_OK;
}

int32_t DenseModel::upload(const void* host, size_t bytes, void** out) {
  KANSO_CUDA_TRY(ctx, cudaMalloc(out, std::max<size_t>(bytes, 16)), "weights");
  owned.push_back(*out);
  KANSO_CUDA_TRY(ctx, cudaMemcpy(*out, host, bytes, cudaMemcpyHostToDevice), "weights");
  return KANSO_OK;
}

int32_t DenseModel::vec(const SafeTensors& st, const std::string& name, int64_t n, float** out,
                        std::vector<float>* host) {
  const StTensor* t = nullptr;
  int32_t e = tensor(st, name, {n}, &t);
  if (e) return e;
  std::vector<float> v((size_t)n);
  for (int64_t i = 0; i < n; ++i) v[(size_t)i] = st_value(*t, i);
  if (out && (e = upload(v.data(), v.size() * 4, (void**)out))) return e;
  if (host) *host = std::move(v);
  return KANSO_OK;
}

int32_t DenseModel::mat_rows(const std::vector<const StTensor*>& parts, int64_t rows,
                             int64_t groups, int64_t cols, bool f32,
                             const std::function<int64_t(int64_t)>& source, DenseMat* out) {
  const int64_t ld = round_up8(cols);
  const size_t es = f32 ? 4 : 2;
  std::vector<uint8_t> host((size_t)(rows * ld) * es, 0);
  std::vector<std::pair<const StTensor*, int64_t>> at;  // row of the parts -> (part, row in it)
  for (const StTensor* t : parts)
    for (int64_t i = 0; i < t->shape[0]; ++i) at.emplace_back(t, i);
  for (int64_t r = 0; r < rows; ++r) {
    const int64_t s = source(r);
    if (s < 0) continue;
    const StTensor* t = at[(size_t)s].first;
    const int64_t first = at[(size_t)s].second * cols;
    uint8_t* dst = host.data() + (size_t)(r * ld) * es;
    if (!f32 && t->type == StType::BF16)
      std::memcpy(dst, t->data + 2 * first, (size_t)cols * 2);
    else
      for (int64_t c = 0; c < cols; ++c) put_value(dst + es * c, f32, st_value(*t, first + c));
  }
  out->rows = rows / groups;
  out->cols = cols;
  out->ld = ld;
  out->groups = groups;
  return upload(host.data(), host.size(), &out->w);
}

int32_t DenseModel::mat(const std::vector<const StTensor*>& parts, int64_t groups, int64_t cols,
                        bool f32, DenseMat* out) {
  int64_t rows = 0;
  for (const StTensor* t : parts) rows += t->shape[0];
  return mat_rows(parts, rows, groups, cols, f32, [](int64_t r) { return r; }, out);
}

int32_t DenseModel::mat_transposed(const StTensor* t, int64_t block, int64_t cols, bool f32,
                                   DenseMat* out) {
  const int64_t groups = t->shape[0] / block, ld = round_up8(block);
  const size_t es = f32 ? 4 : 2;
  std::vector<uint8_t> host((size_t)(groups * cols * ld) * es, 0);
  for (int64_t g = 0; g < groups; ++g)
    for (int64_t b = 0; b < block; ++b)
      for (int64_t c = 0; c < cols; ++c)
        put_value(host.data() + (size_t)((g * cols + c) * ld + b) * es, f32,
                  st_value(*t, (g * block + b) * cols + c));
  out->rows = cols;
  out->cols = block;
  out->ld = ld;
  out->groups = groups;
  return upload(host.data(), host.size(), &out->w);
}

int32_t DenseModel::make_ws(int64_t rows, const std::vector<Room>& parts) {
  cudaStreamSynchronize(ctx->stream);
  if (ws) cudaFree(ws);
  ws = nullptr;
  ws_rows = 0;
  size_t total = 0;
  for (const Room& b : parts) total += (b.bytes + 255) & ~(size_t)255;
  KANSO_CUDA_TRY(ctx, cudaMalloc(&ws, std::max<size_t>(total, 256)), "workspace");
  KANSO_CUDA_TRY(ctx, cudaMemsetAsync(ws, 0, total, ctx->stream), "workspace");
  uint8_t* at = static_cast<uint8_t*>(ws);
  for (const Room& b : parts) {
    *b.p = at;
    at += (b.bytes + 255) & ~(size_t)255;
  }
  ws_rows = rows;
  return KANSO_OK;
}

int32_t DenseModel::logits_of_rows(const DenseMat& head, const float* norm, float eps,
                                   const float* x, void* xe, const DenseStep& s,
                                   float* logits_dev) {
  if (!s.n_want) return KANSO_OK;
  int32_t st;
  if (s.n_want <= GEMV_MAX_T) {
    GemvSource g;
    g.x = x;
    g.eps = eps;
    g.final_w = norm;
    g.row_index = s.want;
    return launch_gemv(ctx, compute, head, g, logits_dev, head.rows, (int)s.n_want);
  }
  // wanted rows in portions of the workspace (a row may be asked for more than once)
  int splits = 1;
  for (int64_t i = 0; i < s.n_want; i += s.T) {
    const int64_t n = std::min(s.T, s.n_want - i);
    if ((st = launch_norm_rows(ctx, compute, x, head.cols, s.want ? s.want + i : nullptr, norm, eps,
                               xe, head.ld, n)))
      return st;
    GemmRows hr;
    hr.T = n;
    if ((st = launch_gemm(ctx, compute, head, xe, logits_dev + i * head.rows, head.rows, hr, 1,
                          &splits, 0)))
      return st;
  }
  return KANSO_OK;
}

int32_t DenseModel::create_pool(uint32_t num_blocks, uint32_t num_slots, kanso_cuda_kv** out) {
  const std::vector<kanso_kv_layer> l = cache_layers();
  return kanso_cuda_kv_create_layers(ctx, (uint32_t)l.size(), l.data(), num_blocks, block_size(),
                                     kv_type(), num_slots, out);
}

int32_t DenseModel::check_pool(const kanso_cuda_kv* kv) {
  const std::vector<kanso_kv_layer> l = cache_layers();
  bool ok = kv->kv_type == kv_type() && kv->dense.size() == l.size();
  for (size_t i = 0; ok && i < l.size(); ++i) {
    const KvDenseLayer& d = kv->dense[i];
    const KvStateLayer& s = kv->state[i];
    ok = d.kv_heads == l[i].kv_heads && d.k_dim == l[i].k_dim && d.v_dim == l[i].v_dim &&
         s.heads == l[i].state_heads && s.dim == l[i].state_dim && s.vdim == l[i].state_vdim;
  }
  return ok ? KANSO_OK
            : fail(ctx, KANSO_ERR_SHAPE, "the pool's geometry or element type is not the model's");
}

int32_t DenseModel::decode_device(kanso_cuda_kv* kv, const uint32_t* tokens,
                                  const uint32_t* positions, const uint32_t*,
                                  const uint32_t* tables, const uint32_t*,
                                  const uint32_t* state_slots, uint32_t B, uint32_t max_blocks,
                                  uint32_t max_ctx, int32_t act_mode, float* logits_dev) {
  if (act_mode != KANSO_ACT_F32)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "decode_step: quantised activations need quantised "
                                            "weights");
  const int32_t st = check_pool(kv);
  if (st) return st;
  if (!state_slots && has_state() && B > kv->num_slots)
    return fail(ctx, KANSO_ERR_SHAPE, "decode_step: %u sequences, %u state slots", B,
                kv->num_slots);
  DenseStep s;
  s.T = s.S = B;
  s.tokens = tokens;
  s.map.positions = positions;  // a token's slot is where the table places its position
  s.map.tables = tables;
  s.map.max_blocks = max_blocks;
  s.n_want = B;
  s.one_each = true;
  s.max_keys = max_ctx;
  s.n_short = B;
  s.n_short_rows = B;
  s.slots = state_slots;
  return run(kv, s, logits_dev);
}

int32_t DenseModel::forward(kanso_cuda_kv* kv, const StepBatch& b, float* logits_dev) {
  // the prompt kernels' tiles; short queries go row by row
  std::vector<AttnTile> tiles128, tiles64, shorts, longs, long_tiles, runs;
  std::vector<uint32_t> short_rows;
  DenseStep s;
  s.T = b.T;
  s.S = b.S;
  s.n_want = b.n_want;
  s.one_each = true;
  uint32_t row = 0;
  const size_t words = 3 * (size_t)b.T + b.n_want + b.S + (size_t)b.S * b.max_blocks;
  step_in.resize(words);
  uint32_t *tok = step_in.data(), *pos = tok + b.T, *seq = pos + b.T, *want = seq + b.T,
           *slot = want + b.n_want, *tab = slot + b.S;
  for (uint32_t i = 0; i < b.S; ++i) {
    const uint32_t n = b.query_lens[i], c = b.context_lens[i], p0 = c - n;
    s.one_each = s.one_each && n == 1;
    s.use_tiles = s.use_tiles || n >= PROMPT_MIN_ROWS;
    s.max_keys = std::max(s.max_keys, c);
    slot[i] = b.state_slots ? b.state_slots[i] : i;
    for (uint32_t k = 0; k < n; k += 128)
      tiles128.push_back({row + k, std::min(128u, n - k), p0 + k, i});
    for (uint32_t k = 0; k < n; k += 64)
      tiles64.push_back({row + k, std::min(64u, n - k), p0 + k, i});
    if (n < PROMPT_MIN_ROWS) {
      shorts.push_back({row, n, p0, i});
      s.max_short_rows = std::max(s.max_short_rows, n);
      for (uint32_t k = 0; k < n; ++k) short_rows.push_back(row + k);
    } else {
      const uint32_t base = (uint32_t)s.long_keys;
      longs.push_back({row, n, p0, i});
      s.max_long_rows = std::max(s.max_long_rows, n);
      runs.push_back({base, c, i, 0});
      for (uint32_t k = 0; k < n; k += 128)
        long_tiles.push_back({row + k, std::min(128u, n - k), p0 + k, base});
      s.long_keys += c;
    }
    for (uint32_t k = 0; k < n; ++k, ++row) {
      pos[row] = p0 + k;
      seq[row] = i;
    }
  }
  std::memcpy(tok, b.tokens, (size_t)b.T * 4);
  if (b.n_want) std::memcpy(want, b.want, (size_t)b.n_want * 4);
  std::memcpy(tab, b.tables, (size_t)b.S * b.max_blocks * 4);
  static_assert(sizeof(AttnTile) == 16, "four words");
  s.n_tiles128 = (uint32_t)tiles128.size();
  s.n_tiles64 = (uint32_t)tiles64.size();
  s.n_short = (uint32_t)shorts.size();
  s.n_long = (uint32_t)longs.size();
  s.n_long_tiles = (uint32_t)long_tiles.size();
  s.n_short_rows = (int64_t)short_rows.size();
  // one array of tiles: by 128, by 64, portions, long tiles, key runs; then the short rows
  std::vector<AttnTile> all;
  for (const auto* v : {&tiles128, &tiles64, &shorts, &longs, &long_tiles, &runs})
    all.insert(all.end(), v->begin(), v->end());
  const size_t tile_at = (words + 3) & ~(size_t)3, rows_at = tile_at + 4 * all.size();
  step_in.resize(rows_at + short_rows.size());
  std::memcpy(step_in.data() + tile_at, all.data(), all.size() * sizeof(AttnTile));
  std::copy(short_rows.begin(), short_rows.end(), step_in.begin() + rows_at);
  int32_t st = model_inputs(this, step_in.size());
  if (st) return st;
  KANSO_CUDA_TRY(ctx,
                 cudaMemcpyAsync(d_in, step_in.data(), step_in.size() * 4, cudaMemcpyHostToDevice,
                                 ctx->stream),
                 "h2d");
  s.tokens = d_in;
  s.map.positions = d_in + b.T;
  s.map.row_seq = d_in + 2 * (size_t)b.T;
  s.want = d_in + 3 * (size_t)b.T;
  s.slots = s.want + b.n_want;
  s.map.tables = s.slots + b.S;
  s.map.max_blocks = b.max_blocks;
  s.tiles128 = reinterpret_cast<const AttnTile*>(d_in + tile_at);
  s.tiles64 = s.tiles128 + s.n_tiles128;
  s.portions = s.tiles64 + s.n_tiles64;
  s.long_tiles = s.portions + s.n_short + s.n_long;
  s.key_runs = s.long_tiles + s.n_long_tiles;
  s.short_rows = d_in + rows_at;
  return run(kv, s, logits_dev);
}

}  // namespace kanso
