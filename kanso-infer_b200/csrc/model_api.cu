// Entry points that work on any model class: the registry and loading from a folder, the pool of
// a model, the decode step and the ragged step with host arrays.
#include <algorithm>
#include <cstring>
#include <fstream>
#include <sstream>

#include "model.h"

namespace kanso {

static std::vector<ModelClass>& registry() {
  static std::vector<ModelClass> r;
  return r;
}
ModelRegistrar::ModelRegistrar(const ModelClass& c) { registry().push_back(c); }

// dir/config.json and the class its "architecture" names.
static int32_t open_config(kanso_cuda_ctx* ctx, const std::string& dir, Json* config,
                           const ModelClass** cls) {
  const std::string path = dir + "/config.json";
  std::ifstream in(path, std::ios::binary);
  if (!in) return fail(ctx, KANSO_ERR_CONFIG, "cannot open '%s'", path.c_str());
  std::stringstream ss;
  ss << in.rdbuf();
  const std::string text = ss.str();
  if (!JsonReader(text.data(), text.size()).parse(config) || config->kind != Json::OBJ)
    return fail(ctx, KANSO_ERR_CONFIG, "'%s' is not a JSON object", path.c_str());
  const Json* arch = config->find("architecture");
  if (!arch || arch->kind != Json::STR)
    return fail(ctx, KANSO_ERR_CONFIG, "'%s' has no \"architecture\"", path.c_str());
  std::string known;
  for (const ModelClass& c : registry()) {
    if (arch->str == c.architecture) {
      *cls = &c;
      return KANSO_OK;
    }
    known += (known.empty() ? "" : ", ") + std::string(c.architecture);
  }
  return fail(ctx, KANSO_ERR_CONFIG, "unknown architecture '%s' (this library loads: %s)",
              arch->str.c_str(), known.c_str());
}

int32_t model_inputs(kanso_cuda_model* m, size_t words) {
  if (words <= m->d_in_cap) return KANSO_OK;
  cudaStreamSynchronize(m->ctx->stream);
  if (m->d_in) cudaFree(m->d_in);
  m->d_in = nullptr;
  m->d_in_cap = 0;
  const size_t want = words + words / 2 + 256;
  KANSO_CUDA_TRY(m->ctx, cudaMalloc((void**)&m->d_in, want * 4), "step inputs");
  m->d_in_cap = want;
  return KANSO_OK;
}

int32_t model_logits(kanso_cuda_model* m, size_t rows) {
  if (rows <= m->logits_cap) return KANSO_OK;
  cudaStreamSynchronize(m->ctx->stream);
  if (m->logits) cudaFree(m->logits);
  m->logits = nullptr;
  m->logits_cap = 0;
  KANSO_CUDA_TRY(m->ctx, cudaMalloc((void**)&m->logits, rows * m->vocab_size() * 4), "logits");
  m->logits_cap = rows;
  return KANSO_OK;
}

int32_t check_step(kanso_cuda_model* m, const kanso_cuda_kv* kv, const StepBatch& b) {
  kanso_cuda_ctx* ctx = m->ctx;
  int32_t st = m->check_pool(kv);
  if (st) return st;
  const uint32_t bs = kv->block_size, limit = m->max_query_len(), window = m->max_window();
  uint64_t T = 0;
  for (uint32_t s = 0; s < b.S; ++s) {
    const uint32_t q = b.query_lens[s], c = b.context_lens[s];
    if (q == 0 || q > c)
      return fail(ctx, KANSO_ERR_SHAPE, "step: sequence %u brings %u of %u tokens", s, q, c);
    if (limit && q > limit)
      return fail(ctx, KANSO_ERR_UNSUPPORTED,
                  "step: a %s model takes %u token(s) of a sequence per step, not %u",
                  m->architecture(), limit, q);
    if (m->max_positions() && c > m->max_positions())
      return fail(ctx, KANSO_ERR_SHAPE, "step: position %u beyond max_seq_len %u", c - 1,
                  m->max_positions());
    const uint32_t need = (c + bs - 1) / bs;
    if (need > b.max_blocks)
      return fail(ctx, KANSO_ERR_SHAPE,
                  "step: sequence %u attends %u tokens but its block table has %u of the %u blocks "
                  "needed", s, c, b.max_blocks, need);
    // entries wholly behind every window are never read and may be stale
    const uint32_t first_pos = c - q;
    const uint32_t from = window && first_pos + 1 > window ? (first_pos + 1 - window) / bs : 0;
    for (uint32_t i = from; i < need; ++i)
      if (b.tables[(size_t)s * b.max_blocks + i] >= kv->num_blocks)
        return fail(ctx, KANSO_ERR_SHAPE, "Physical block index %u out of bounds (%u)",
                    b.tables[(size_t)s * b.max_blocks + i], kv->num_blocks);
    T += q;
  }
  if (T != b.T) return fail(ctx, KANSO_ERR_SHAPE, "step: %u tokens, queries sum to %llu", b.T,
                            (unsigned long long)T);
  for (uint32_t t = 0; t < b.T; ++t)
    if (b.tokens[t] >= m->vocab_size())
      return fail(ctx, KANSO_ERR_SHAPE, "step: token id %u out of range (vocab %u)", b.tokens[t],
                  m->vocab_size());
  if (m->has_state()) {
    std::vector<bool> taken(kv->num_slots);
    for (uint32_t s = 0; s < b.S; ++s) {
      const uint32_t slot = b.state_slots ? b.state_slots[s] : s;
      if (slot >= kv->num_slots || taken[slot])
        return fail(ctx, KANSO_ERR_SHAPE, "step: state slot %u of sequence %u (the pool has %u)%s",
                    slot, s, kv->num_slots, slot < kv->num_slots ? " is taken" : "");
      taken[slot] = true;
    }
  }
  for (uint32_t i = 0; i < b.n_want; ++i)
    if (b.want[i] >= b.T)
      return fail(ctx, KANSO_ERR_SHAPE, "step: logits of row %u of %u", b.want[i], b.T);
  return KANSO_OK;
}

int32_t run_step(kanso_cuda_model* m, kanso_cuda_kv* kv, const StepBatch& b) {
  int32_t st = check_step(m, kv, b);
  if (!st && b.n_want) st = model_logits(m, b.n_want);
  return st ? st : m->forward(kv, b, m->logits);
}

}  // namespace kanso

using namespace kanso;

kanso_cuda_model::~kanso_cuda_model() {
  if (d_in) cudaFree(d_in);
  if (logits) cudaFree(logits);
}

extern "C" {

int32_t kanso_cuda_model_destroy(kanso_cuda_model* m) {
  if (!m) return KANSO_OK;
  cudaDeviceSynchronize();  // the context may already be destroyed
  delete m;
  return KANSO_OK;
}

int32_t kanso_cuda_model_describe(const char* dir, char* out, size_t out_bytes) {
  if (!dir || !out || !out_bytes)
    return fail(nullptr, KANSO_ERR_CONFIG, "model_describe: NULL argument");
  Json config;
  const ModelClass* cls = nullptr;
  std::string text;
  int32_t st = open_config(nullptr, dir, &config, &cls);
  if (!st) st = cls->describe(nullptr, config, &text);
  if (st) return st;
  if (text.size() + 1 > out_bytes)
    return fail(nullptr, KANSO_ERR_SHAPE, "model_describe: %zu bytes needed", text.size() + 1);
  std::memcpy(out, text.c_str(), text.size() + 1);
  return KANSO_OK;
}

int32_t kanso_cuda_model_load(kanso_cuda_ctx* ctx, const char* dir, int32_t compute,
                              kanso_cuda_model** out) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "model_load: ctx is NULL");
  if (!dir || !out) return fail(ctx, KANSO_ERR_CONFIG, "model_load: NULL argument");
  *out = nullptr;
  if (compute != KANSO_COMPUTE_BF16 && compute != KANSO_COMPUTE_F32)
    return fail(ctx, KANSO_ERR_CONFIG, "model_load: unknown number format %d", compute);
  Json config;
  const ModelClass* cls = nullptr;
  int32_t st = open_config(ctx, dir, &config, &cls);
  return st ? st : cls->load(ctx, config, dir, compute, out);
}

int32_t kanso_cuda_model_create_pool(kanso_cuda_model* m, uint32_t num_blocks,
                                     kanso_cuda_kv** out) {
  if (!m) return fail(nullptr, KANSO_ERR_CONFIG, "model_create_pool: model is NULL");
  // no more sequences than pages can be live
  return kanso_cuda_model_create_pool_slots(m, num_blocks, std::min(num_blocks, 256u), out);
}

int32_t kanso_cuda_model_create_pool_slots(kanso_cuda_model* m, uint32_t num_blocks,
                                           uint32_t num_slots, kanso_cuda_kv** out) {
  if (!m) return fail(nullptr, KANSO_ERR_CONFIG, "model_create_pool: model is NULL");
  if (!out) return fail(m->ctx, KANSO_ERR_CONFIG, "model_create_pool: out is NULL");
  return m->create_pool(num_blocks, num_slots, out);
}

int32_t kanso_cuda_forward_step(kanso_cuda_ctx* ctx, kanso_cuda_model* m, kanso_cuda_kv* kv,
                                const uint32_t* tokens, const uint32_t* query_lens,
                                const uint32_t* context_lens, const uint32_t* block_tables,
                                uint32_t S, uint32_t max_blocks, const uint32_t* want,
                                uint32_t n_want, float* logits_out) {
  return kanso_cuda_forward_step_slots(ctx, m, kv, tokens, query_lens, context_lens, block_tables,
                                       nullptr, S, max_blocks, want, n_want, logits_out);
}

int32_t kanso_cuda_forward_step_slots(kanso_cuda_ctx* ctx, kanso_cuda_model* m, kanso_cuda_kv* kv,
                                      const uint32_t* tokens, const uint32_t* query_lens,
                                      const uint32_t* context_lens, const uint32_t* block_tables,
                                      const uint32_t* state_slots, uint32_t S, uint32_t max_blocks,
                                      const uint32_t* want, uint32_t n_want, float* logits_out) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "forward_step: ctx is NULL");
  if (!m || !kv) return fail(ctx, KANSO_ERR_SHAPE, "forward_step: model or pool is NULL");
  if (S == 0) return KANSO_OK;
  if (!tokens || !query_lens || !context_lens || !block_tables || !max_blocks ||
      (n_want && (!want || !logits_out)))
    return fail(ctx, KANSO_ERR_SHAPE, "forward_step: NULL argument");
  StepBatch b;
  b.S = S;
  for (uint32_t s = 0; s < S; ++s) b.T += query_lens[s];
  b.max_blocks = max_blocks;
  b.tokens = tokens;
  b.query_lens = query_lens;
  b.context_lens = context_lens;
  b.tables = block_tables;
  b.state_slots = state_slots;
  b.want = want;
  b.n_want = n_want;
  int32_t st = run_step(m, kv, b);
  if (st) return st;
  if (n_want)
    KANSO_CUDA_TRY(ctx,
                   cudaMemcpyAsync(logits_out, m->logits, (size_t)n_want * m->vocab_size() * 4,
                                   cudaMemcpyDeviceToHost, ctx->stream),
                   "d2h");
  return kanso_cuda_sync(ctx);
}

int32_t kanso_cuda_decode_step_device(kanso_cuda_ctx* ctx, kanso_cuda_model* m, kanso_cuda_kv* kv,
                                      const uint32_t* tokens, const uint32_t* positions,
                                      const uint32_t* slots, const uint32_t* block_tables,
                                      const uint32_t* context_lens, uint32_t B,
                                      uint32_t max_blocks, uint32_t max_ctx, int32_t act_mode,
                                      float* logits_dev) {
  return kanso_cuda_decode_step_device_slots(ctx, m, kv, tokens, positions, slots, block_tables,
                                             context_lens, nullptr, B, max_blocks, max_ctx,
                                             act_mode, logits_dev);
}

int32_t kanso_cuda_decode_step_device_slots(kanso_cuda_ctx* ctx, kanso_cuda_model* m,
                                            kanso_cuda_kv* kv, const uint32_t* tokens,
                                            const uint32_t* positions, const uint32_t* slots,
                                            const uint32_t* block_tables,
                                            const uint32_t* context_lens,
                                            const uint32_t* state_slots, uint32_t B,
                                            uint32_t max_blocks, uint32_t max_ctx,
                                            int32_t act_mode, float* logits_dev) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "decode_step: ctx is NULL");
  if (!m || !kv) return fail(ctx, KANSO_ERR_SHAPE, "decode_step: model or pool is NULL");
  if (B == 0) return KANSO_OK;
  return m->decode_device(kv, tokens, positions, slots, block_tables, context_lens, state_slots, B,
                          max_blocks, max_ctx, act_mode, logits_dev);
}

int32_t kanso_cuda_decode_step(kanso_cuda_ctx* ctx, kanso_cuda_model* m, kanso_cuda_kv* kv,
                               const uint32_t* tokens, const uint32_t* positions,
                               const uint32_t* slots, const uint32_t* block_tables,
                               const uint32_t* context_lens, uint32_t B, uint32_t max_blocks,
                               int32_t act_mode, float* logits_out) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "decode_step: ctx is NULL");
  if (!m || !kv) return fail(ctx, KANSO_ERR_SHAPE, "decode_step: model or pool is NULL");
  if (B == 0) return KANSO_OK;
  if (!tokens || !positions || !slots || !block_tables || !context_lens || !logits_out)
    return fail(ctx, KANSO_ERR_SHAPE, "decode_step: NULL argument");
  if (max_blocks == 0) return fail(ctx, KANSO_ERR_SHAPE, "decode_step: max_blocks is 0");
  // host-side checks the reference makes before touching the pool
  const uint32_t bs = kv->block_size, vocab = m->vocab_size();
  uint32_t max_ctx = 0;
  for (uint32_t s = 0; s < B; ++s) {
    if (tokens[s] >= vocab)
      return fail(ctx, KANSO_ERR_SHAPE, "decode_step: token id %u out of range (vocab %u)",
                  tokens[s], vocab);
    if (m->max_positions() && positions[s] >= m->max_positions())
      return fail(ctx, KANSO_ERR_SHAPE, "decode_step: position %u beyond max_seq_len %u",
                  positions[s], m->max_positions());
    if ((uint64_t)slots[s] >= (uint64_t)kv->num_blocks * bs)
      return fail(ctx, KANSO_ERR_SHAPE, "Slot %u out of bounds for %u blocks of size %u", slots[s],
                  kv->num_blocks, bs);
    uint32_t ctxlen = context_lens[s];
    if (ctxlen == 0 || (ctxlen + bs - 1) / bs > max_blocks)
      // src/model.rs:92-101: a table shorter than ceil(ctx/bs) is an error, never a clamp
      return fail(ctx, KANSO_ERR_SHAPE,
                  "forward_batch: sequence %u attends %u tokens but its block table has %u of the "
                  "%u blocks needed",
                  s, ctxlen, max_blocks, (ctxlen + bs - 1) / bs);
    for (uint32_t b = 0; b < (ctxlen + bs - 1) / bs; ++b)
      if (block_tables[(size_t)s * max_blocks + b] >= kv->num_blocks)
        return fail(ctx, KANSO_ERR_SHAPE, "Physical block index %u out of bounds (%u)",
                    block_tables[(size_t)s * max_blocks + b], kv->num_blocks);
    if (ctxlen > max_ctx) max_ctx = ctxlen;
  }
  const size_t nb = (size_t)B * 4, tb = (size_t)B * max_blocks * 4, lb = (size_t)B * vocab * 4;
  int32_t st = model_inputs(m, 4 * (size_t)B + (size_t)B * max_blocks);
  if (!st) st = model_logits(m, B);
  if (!st) st = ctx_pinned(ctx, 4 * nb + tb + lb);
  if (st) return st;
  char* ph = (char*)ctx->pinned;
  std::memcpy(ph, tokens, nb);
  std::memcpy(ph + nb, positions, nb);
  std::memcpy(ph + 2 * nb, slots, nb);
  std::memcpy(ph + 3 * nb, context_lens, nb);
  std::memcpy(ph + 4 * nb, block_tables, tb);
  cudaStream_t s = ctx->stream;
  KANSO_CUDA_TRY(ctx, cudaMemcpyAsync(m->d_in, ph, 4 * nb + tb, cudaMemcpyHostToDevice, s), "h2d");
  st = m->decode_device(kv, m->d_in, m->d_in + B, m->d_in + 2 * B, m->d_in + 4 * B, m->d_in + 3 * B,
                        nullptr, B, max_blocks, max_ctx, act_mode, m->logits);
  if (st) return st;
  char* pl = ph + 4 * nb + tb;
  KANSO_CUDA_TRY(ctx, cudaMemcpyAsync(pl, m->logits, lb, cudaMemcpyDeviceToHost, s), "d2h");
  if ((st = kanso_cuda_sync(ctx))) return st;
  std::memcpy(logits_out, pl, lb);
  return KANSO_OK;
}

}  // extern "C"
