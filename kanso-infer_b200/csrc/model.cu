// Decode step of a Llama-architecture model on the cuda backend:
// Model::forward_decode_step / forward_batch on a pure-decode batch
// (src/model.rs:1101-1231,1418-1740), one token per sequence.
#include <cmath>
#include <cstring>

#include "glue.cuh"
#include "model.h"

namespace kanso {
int32_t launch_paged_attention(kanso_cuda_ctx* ctx, const kanso_cuda_kv* kv, uint32_t layer,
                               const float* q, const uint32_t* tables, const uint32_t* lens,
                               float* out, const kanso_paged_attention_params* p,
                               uint32_t max_ctx_hint, const PaDecodeFusion* fusion);
int32_t tc_matmul_multi(kanso_cuda_ctx* ctx, int32_t dtype, int nseg, const void* const* w,
                        float* const* y, const int64_t* rows, const float* x, const float* x2,
                        const float* norm_w, float eps, const float* resid, int64_t M, int64_t K,
                        bool* handled, const void* prepacked);

// Embedding rows of a Q8_0 table (src/weights.rs:50-57), bit-exact d * (f32)q.
__global__ void model_embed_kernel(const uint8_t* __restrict__ w, const uint32_t* __restrict__ ids,
                                   float* __restrict__ out, int64_t rows, int cols, int* status) {
  int t = blockIdx.x;
  uint32_t id = ids[t];
  if (id >= rows) {
    if (threadIdx.x == 0) atomicOr(status, DEV_BAD_INDEX);
    id = 0;
  }
  const uint8_t* row = w + (int64_t)id * (cols / 32) * Q8_BYTES;
  for (int i = threadIdx.x; i < cols; i += blockDim.x) {
    const uint8_t* blk = row + (i >> 5) * Q8_BYTES;
    float d = f16_bits_to_f32(blk[0] | (blk[1] << 8));
    out[(int64_t)t * cols + i] = __fmul_rn(d, (float)(int8_t)blk[2 + (i & 31)]);
  }
}
}  // namespace kanso

struct ModelLin {
  void* dev = nullptr;
  int32_t dtype = 0;
  int64_t rows = 0, cols = 0;
};

struct LlamaModel final : kanso_cuda_model {
  kanso_model_config cfg{};
  struct Layer {
    ModelLin w[7];
    float* attn_norm = nullptr;
    float* ffn_norm = nullptr;
  };
  std::vector<Layer> layers;
  ModelLin token_embd, output;
  float* final_norm = nullptr;
  // RoPE table rows [max_seq_len][head_dim/2], built on the host like build_rope_table
  float* rope_cos = nullptr;
  float* rope_sin = nullptr;
  int rope_len = 0;
  // workspace for B sequences
  uint32_t ws_B = 0;
  float *hidden = nullptr, *normed = nullptr, *qkv = nullptr, *attn = nullptr, *proj = nullptr,
        *gate = nullptr, *up = nullptr, *act = nullptr;
  std::vector<uint32_t> step_in;  // host image of a step's inputs

  ~LlamaModel() override;
  const char* architecture() const override { return "llama"; }
  uint32_t vocab_size() const override { return cfg.vocab_size; }
  uint32_t num_layers() const override { return cfg.num_hidden_layers; }
  uint32_t block_size() const override { return cfg.block_size ? cfg.block_size : 16; }
  uint32_t max_positions() const override { return cfg.max_seq_len; }
  uint32_t max_query_len() const override { return 1; }  // its step is the decode step
  int32_t create_pool(uint32_t num_blocks, uint32_t num_slots, kanso_cuda_kv** out) override;
  int32_t check_pool(const kanso_cuda_kv* kv) override;
  int32_t decode_device(kanso_cuda_kv* kv, const uint32_t* tokens, const uint32_t* positions,
                        const uint32_t* slots, const uint32_t* tables,
                        const uint32_t* context_lens, const uint32_t* state_slots, uint32_t B,
                        uint32_t max_blocks, uint32_t max_ctx, int32_t act_mode,
                        float* logits_dev) override;
  int32_t forward(kanso_cuda_kv* kv, const kanso::StepBatch& b, float* logits_dev) override;
};

using namespace kanso;

static void free_ws(LlamaModel* m) {
  for (float** p : {&m->hidden, &m->normed, &m->qkv, &m->attn, &m->proj, &m->gate, &m->up,
                    &m->act}) {
    if (*p) cudaFree(*p);
    *p = nullptr;
  }
  m->ws_B = 0;
}

static int32_t ensure_ws(LlamaModel* m, uint32_t B) {
  kanso_cuda_ctx* ctx = m->ctx;
  if (B <= m->ws_B) return KANSO_OK;
  cudaStreamSynchronize(ctx->stream);
  free_ws(m);
  const auto& c = m->cfg;
  const uint32_t hd = c.hidden_size / c.num_attention_heads;
  const size_t qkv_w = (size_t)(c.num_attention_heads + 2 * c.num_key_value_heads) * hd;
  struct {
    float** p;
    size_t n;
  } fb[] = {{&m->hidden, (size_t)B * c.hidden_size},
            {&m->normed, (size_t)B * c.hidden_size},
            {&m->qkv, (size_t)B * qkv_w},
            {&m->attn, (size_t)B * c.num_attention_heads * hd},
            {&m->proj, (size_t)B * c.hidden_size},
            {&m->gate, (size_t)B * c.intermediate_size},
            {&m->up, (size_t)B * c.intermediate_size},
            {&m->act, (size_t)B * c.intermediate_size}};
  for (auto& b : fb) KANSO_CUDA_TRY(ctx, cudaMalloc((void**)b.p, b.n * sizeof(float)), "workspace");
  m->ws_B = B;
  return KANSO_OK;
}

// Up to three projections of the same activations in one tensor-core GEMM launch (9..128
// activation rows), with rmsnorm (norm_w) or the SwiGLU product (x2) folded into the activation
// pack and the residual add into the epilogue (resid). *handled = false, nothing launched, when the
// weights or shapes are outside that kernel's range: the caller then runs the pieces singly.
static int32_t lin_multi(kanso_cuda_ctx* ctx, int n, const ModelLin* const* l, float* const* y,
                         const float* x, const float* x2, const float* norm_w, float eps,
                         const float* resid, int64_t M, int32_t act_mode, bool* handled,
                         const void* prepacked = nullptr) {
  *handled = false;
  if (act_mode != KANSO_ACT_F32 || M <= 8 || M > 128) return KANSO_OK;
  const void* w[3];
  int64_t rows[3];
  for (int i = 0; i < n; ++i) {
    if (!l[i]->dev || l[i]->dtype != l[0]->dtype || l[i]->cols != l[0]->cols) return KANSO_OK;
    w[i] = l[i]->dev;
    rows[i] = l[i]->rows;
  }
  if (l[0]->dtype != KANSO_DTYPE_Q8_0 && l[0]->dtype != KANSO_DTYPE_Q4_K) return KANSO_OK;
  return tc_matmul_multi(ctx, l[0]->dtype, n, w, y, rows, x, x2, norm_w, eps, resid, M,
                         l[0]->cols, handled, prepacked);
}

static int32_t lin(kanso_cuda_ctx* ctx, const ModelLin& l, const float* x, float* y, int64_t M,
                   int32_t act_mode) {
  if (!l.dev) return fail(ctx, KANSO_ERR_CONFIG, "decode_step: a projection weight is not set");
  return matmul_dispatch(ctx, l.dtype, l.dev, x, y, M, l.rows, l.cols, act_mode);
}

extern "C" {

int32_t kanso_cuda_model_create(kanso_cuda_ctx* ctx, const kanso_model_config* cfg,
                                kanso_cuda_model** out) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "model_create: ctx is NULL");
  if (!cfg || !out) return fail(ctx, KANSO_ERR_CONFIG, "model_create: NULL argument");
  *out = nullptr;
  if (!cfg->hidden_size || !cfg->num_attention_heads || !cfg->num_key_value_heads ||
      !cfg->num_hidden_layers || !cfg->intermediate_size || !cfg->vocab_size || !cfg->max_seq_len)
    return fail(ctx, KANSO_ERR_CONFIG, "model_create: every dimension must be non-zero");
  if (cfg->hidden_size % cfg->num_attention_heads ||
      cfg->num_attention_heads % cfg->num_key_value_heads)
    return fail(ctx, KANSO_ERR_CONFIG,
                "model_create: hidden %u / heads %u / kv heads %u do not divide", cfg->hidden_size,
                cfg->num_attention_heads, cfg->num_key_value_heads);
  const uint32_t hd = cfg->hidden_size / cfg->num_attention_heads;
  if (hd % 2) return fail(ctx, KANSO_ERR_CONFIG, "model_create: head_dim %u is odd", hd);
  auto* m = new LlamaModel;
  m->ctx = ctx;
  m->cfg = *cfg;
  m->layers.resize(cfg->num_hidden_layers);
  // build_rope_table (src/model.rs:698-719), on the host with the same libm calls
  const uint32_t half = hd / 2;
  m->rope_len = (int)cfg->max_seq_len;
  std::vector<float> c((size_t)m->rope_len * half), s((size_t)m->rope_len * half), freq(half);
  for (uint32_t j = 0; j < half; ++j)
    freq[j] = std::pow(cfg->rope_theta, -2.0f * (float)j / (float)hd);
  for (int p = 0; p < m->rope_len; ++p)
    for (uint32_t j = 0; j < half; ++j) {
      float a = (float)p * freq[j];
      c[(size_t)p * half + j] = std::cos(a);
      s[(size_t)p * half + j] = std::sin(a);
    }
  cudaError_t e = cudaMalloc((void**)&m->rope_cos, c.size() * 4);
  if (e == cudaSuccess) e = cudaMalloc((void**)&m->rope_sin, s.size() * 4);
  if (e == cudaSuccess) e = cudaMemcpy(m->rope_cos, c.data(), c.size() * 4, cudaMemcpyHostToDevice);
  if (e == cudaSuccess) e = cudaMemcpy(m->rope_sin, s.data(), s.size() * 4, cudaMemcpyHostToDevice);
  if (e != cudaSuccess) {
    kanso_cuda_model_destroy(m);
    return cuda_fail(ctx, e, "model_create: rope table");
  }
  *out = m;
  return KANSO_OK;
}

int32_t kanso_cuda_model_set_weight(kanso_cuda_model* model, uint32_t layer, int32_t which,
                                    const void* host_bytes, size_t nbytes, int32_t dtype,
                                    int64_t rows, int64_t cols) {
  if (!model) return fail(nullptr, KANSO_ERR_CONFIG, "model_set_weight: model is NULL");
  kanso_cuda_ctx* ctx = model->ctx;
  auto* m = dynamic_cast<LlamaModel*>(model);
  if (!m)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "model_set_weight: a %s model loads from its folder",
                model->architecture());
  const auto& c = m->cfg;
  const uint32_t hd = c.hidden_size / c.num_attention_heads;
  int64_t er, ec;
  switch (which) {
    case KANSO_W_ATTN_Q: er = (int64_t)c.num_attention_heads * hd; ec = c.hidden_size; break;
    case KANSO_W_ATTN_K:
    case KANSO_W_ATTN_V: er = (int64_t)c.num_key_value_heads * hd; ec = c.hidden_size; break;
    case KANSO_W_ATTN_OUTPUT: er = c.hidden_size; ec = (int64_t)c.num_attention_heads * hd; break;
    case KANSO_W_FFN_GATE:
    case KANSO_W_FFN_UP: er = c.intermediate_size; ec = c.hidden_size; break;
    case KANSO_W_FFN_DOWN: er = c.hidden_size; ec = c.intermediate_size; break;
    case KANSO_W_TOKEN_EMBD:
    case KANSO_W_OUTPUT: er = c.vocab_size; ec = c.hidden_size; break;
    default: return fail(ctx, KANSO_ERR_CONFIG, "model_set_weight: unknown tensor %d", which);
  }
  if (rows != er || cols != ec)
    return fail(ctx, KANSO_ERR_SHAPE, "model_set_weight: tensor %d is [%lld x %lld], config needs [%lld x %lld]",
                which, (long long)rows, (long long)cols, (long long)er, (long long)ec);
  if (which < KANSO_W_TOKEN_EMBD && layer >= m->layers.size())
    return fail(ctx, KANSO_ERR_SHAPE, "Layer index %u out of bounds (%zu)", layer,
                m->layers.size());
  if (which == KANSO_W_TOKEN_EMBD && dtype != KANSO_DTYPE_Q8_0)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "model_set_weight: token_embd must be Q8_0");
  kanso_cuda_weight* tmp = nullptr;
  int32_t st = kanso_cuda_weight_upload(ctx, host_bytes, nbytes, dtype, rows, cols, &tmp);
  if (st) return st;
  ModelLin& dst = which == KANSO_W_TOKEN_EMBD ? m->token_embd
                  : which == KANSO_W_OUTPUT   ? m->output
                                              : m->layers[layer].w[which];
  if (dst.dev) cudaFree(dst.dev);
  dst.dev = tmp->dev;
  dst.dtype = dtype;
  dst.rows = rows;
  dst.cols = cols;
  delete tmp;  // the device buffer now belongs to the model
  return KANSO_OK;
}

int32_t kanso_cuda_model_set_norm(kanso_cuda_model* model, uint32_t layer, int32_t which,
                                  const float* host_weight, int64_t n) {
  if (!model) return fail(nullptr, KANSO_ERR_CONFIG, "model_set_norm: model is NULL");
  kanso_cuda_ctx* ctx = model->ctx;
  auto* m = dynamic_cast<LlamaModel*>(model);
  if (!m)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "model_set_norm: a %s model loads from its folder",
                model->architecture());
  if (n != (int64_t)m->cfg.hidden_size)
    return fail(ctx, KANSO_ERR_SHAPE, "model_set_norm: %lld weights, hidden size is %u",
                (long long)n, m->cfg.hidden_size);
  float** dst;
  if (which == KANSO_NORM_FINAL) {
    dst = &m->final_norm;
  } else if (which == KANSO_NORM_ATTN || which == KANSO_NORM_FFN) {
    if (layer >= m->layers.size())
      return fail(ctx, KANSO_ERR_SHAPE, "Layer index %u out of bounds (%zu)", layer,
                  m->layers.size());
    dst = which == KANSO_NORM_ATTN ? &m->layers[layer].attn_norm : &m->layers[layer].ffn_norm;
  } else {
    return fail(ctx, KANSO_ERR_CONFIG, "model_set_norm: unknown norm %d", which);
  }
  if (!*dst) KANSO_CUDA_TRY(ctx, cudaMalloc((void**)dst, n * 4), "model_set_norm");
  KANSO_CUDA_TRY(ctx, cudaMemcpy(*dst, host_weight, n * 4, cudaMemcpyHostToDevice),
                 "model_set_norm");
  return KANSO_OK;
}

}  // extern "C"

LlamaModel::~LlamaModel() {
  free_ws(this);
  for (auto& l : layers) {
    for (auto& w : l.w)
      if (w.dev) cudaFree(w.dev);
    if (l.attn_norm) cudaFree(l.attn_norm);
    if (l.ffn_norm) cudaFree(l.ffn_norm);
  }
  if (token_embd.dev) cudaFree(token_embd.dev);
  if (output.dev) cudaFree(output.dev);
  if (final_norm) cudaFree(final_norm);
  if (rope_cos) cudaFree(rope_cos);
  if (rope_sin) cudaFree(rope_sin);
}

int32_t LlamaModel::create_pool(uint32_t num_blocks, uint32_t, kanso_cuda_kv** out) {
  return kanso_cuda_kv_create(ctx, cfg.num_hidden_layers, num_blocks, block_size(),
                              cfg.num_key_value_heads, cfg.hidden_size / cfg.num_attention_heads,
                              KANSO_KV_INT8, out);
}

int32_t LlamaModel::check_pool(const kanso_cuda_kv* kv) {
  const uint32_t KH = cfg.num_key_value_heads, hd = cfg.hidden_size / cfg.num_attention_heads;
  if (!kv->dense.empty() || kv->layers < cfg.num_hidden_layers || kv->kv_heads != KH ||
      kv->head_dim != hd)
    return fail(ctx, KANSO_ERR_SHAPE,
                "decode_step: pool geometry (layers %u, kv_heads %u, head_dim %u) does not match "
                "the model (%u, %u, %u)",
                kv->layers, kv->kv_heads, kv->head_dim, cfg.num_hidden_layers, KH, hd);
  return KANSO_OK;
}

// A ragged step of one token per sequence: the decode step; wanted rows are then gathered.
int32_t LlamaModel::forward(kanso_cuda_kv* kv, const StepBatch& b, float* logits_dev) {
  const uint32_t B = b.S, bs = kv->block_size;
  const size_t words = 4 * (size_t)B + (size_t)B * b.max_blocks;
  step_in.resize(words);
  uint32_t* p = step_in.data();
  uint32_t max_ctx = 0;
  for (uint32_t s = 0; s < B; ++s) {
    const uint32_t c = b.context_lens[s], pos = c - 1;
    p[s] = b.tokens[s];
    p[B + s] = pos;
    p[2 * B + s] = b.tables[(size_t)s * b.max_blocks + pos / bs] * bs + pos % bs;
    p[3 * B + s] = c;
    if (c > max_ctx) max_ctx = c;
  }
  std::memcpy(p + 4 * B, b.tables, (size_t)B * b.max_blocks * 4);
  int32_t st = model_inputs(this, words);
  if (!st) st = ctx_stage_dev(ctx, (size_t)B * cfg.vocab_size * 4);
  if (st) return st;
  KANSO_CUDA_TRY(ctx, cudaMemcpyAsync(d_in, p, words * 4, cudaMemcpyHostToDevice, ctx->stream),
                 "h2d");
  float* all = (float*)ctx->stage_dev;
  st = decode_device(kv, d_in, d_in + B, d_in + 2 * B, d_in + 4 * B, d_in + 3 * B, nullptr, B,
                     b.max_blocks, max_ctx, KANSO_ACT_F32, all);
  if (st) return st;
  for (uint32_t i = 0; i < b.n_want; ++i)
    KANSO_CUDA_TRY(ctx,
                   cudaMemcpyAsync(logits_dev + (size_t)i * cfg.vocab_size,
                                   all + (size_t)b.want[i] * cfg.vocab_size,
                                   (size_t)cfg.vocab_size * 4, cudaMemcpyDeviceToDevice,
                                   ctx->stream),
                   "wanted rows");
  return KANSO_OK;
}

int32_t LlamaModel::decode_device(kanso_cuda_kv* kv, const uint32_t* tokens,
                                  const uint32_t* positions, const uint32_t* slots,
                                  const uint32_t* block_tables, const uint32_t* context_lens,
                                  const uint32_t*, uint32_t B, uint32_t max_blocks, uint32_t max_ctx,
                                  int32_t act_mode, float* logits_dev) {
  LlamaModel* m = this;
  const auto& c = m->cfg;
  const uint32_t H = c.num_attention_heads, KH = c.num_key_value_heads;
  const uint32_t hd = c.hidden_size / H, hidden = c.hidden_size, inter = c.intermediate_size;
  int32_t st = check_pool(kv);
  if (st) return st;
  if (!m->token_embd.dev || !m->final_norm)
    return fail(ctx, KANSO_ERR_CONFIG, "decode_step: token_embd / final norm not set");
  if ((st = ensure_ws(m, B))) return st;
  const size_t qw = (size_t)H * hd, kw = (size_t)KH * hd;
  float* q = m->qkv;
  float* k = m->qkv + (size_t)B * qw;
  float* v = k + (size_t)B * kw;
  kanso_paged_attention_params pa{B, H, KH, hd, kv->block_size, max_blocks,
                                  1.0f / std::sqrt((float)hd)};

  model_embed_kernel<<<B, 256, 0, ctx->stream>>>((const uint8_t*)m->token_embd.dev, tokens,
                                                 m->hidden, m->token_embd.rows, (int)hidden,
                                                 ctx->dev_status);
  if ((st = after_launch(ctx, "embed"))) return st;
  const ModelLin& head = m->output.dev ? m->output : m->token_embd;  // tied lm_head

  // RoPE of q and of the new k, and the int8 store of the new K/V rows, run inside the
  // attention kernel. context_lens counts the new token, whose row is slots[seq] and must be
  // where block_tables places position context_len - 1.
  const PaDecodeFusion fusion = {k, v, positions, slots, m->rope_cos, m->rope_sin, m->rope_len};

  // Up to 8 sequences on Q8_0 weights: 5 launches per layer. The norms are folded into the
  // activation staging of the projections that follow them, SiLU*up into ffn_down's, the
  // residual adds into the epilogues, the split-context merge into the attention kernel.
  bool fused = B <= 8 && head.dtype == KANSO_DTYPE_Q8_0;
  for (uint32_t l = 0; l < c.num_hidden_layers && fused; ++l)
    for (const auto& w : m->layers[l].w) fused = fused && w.dev && w.dtype == KANSO_DTYPE_Q8_0;
  if (fused) {
    for (uint32_t l = 0; l < c.num_hidden_layers; ++l) {
      auto& ly = m->layers[l];
      if (!ly.attn_norm || !ly.ffn_norm)
        return fail(ctx, KANSO_ERR_CONFIG, "decode_step: norm weights of layer %u not set", l);
      {
        const void* w3[3] = {ly.w[KANSO_W_ATTN_Q].dev, ly.w[KANSO_W_ATTN_K].dev,
                             ly.w[KANSO_W_ATTN_V].dev};
        float* y3[3] = {q, k, v};
        const int64_t r3[3] = {(int64_t)qw, (int64_t)kw, (int64_t)kw};
        if ((st = stream_fused_q8_0(ctx, 3, w3, y3, r3, m->hidden, nullptr, ly.attn_norm,
                                    c.rms_norm_eps, nullptr, hidden, (int)B, act_mode)))
          return st;
      }
      // RoPE of q and k and the int8 store of the new K/V rows happen inside the attention
      if ((st = launch_paged_attention(ctx, kv, l, q, block_tables, context_lens, m->attn, &pa,
                                       max_ctx, &fusion)))
        return st;
      {
        const void* w1[1] = {ly.w[KANSO_W_ATTN_OUTPUT].dev};
        float* y1[1] = {m->hidden};
        const int64_t r1[1] = {(int64_t)hidden};
        if ((st = stream_fused_q8_0(ctx, 1, w1, y1, r1, m->attn, nullptr, nullptr, 0.f, m->hidden,
                                    qw, (int)B, act_mode)))
          return st;
      }
      {
        const void* w2[2] = {ly.w[KANSO_W_FFN_GATE].dev, ly.w[KANSO_W_FFN_UP].dev};
        float* y2[2] = {m->gate, m->up};
        const int64_t r2[2] = {(int64_t)inter, (int64_t)inter};
        if ((st = stream_fused_q8_0(ctx, 2, w2, y2, r2, m->hidden, nullptr, ly.ffn_norm,
                                    c.rms_norm_eps, nullptr, hidden, (int)B, act_mode)))
          return st;
      }
      {
        const void* w1[1] = {ly.w[KANSO_W_FFN_DOWN].dev};
        float* y1[1] = {m->hidden};
        const int64_t r1[1] = {(int64_t)hidden};
        if ((st = stream_fused_q8_0(ctx, 1, w1, y1, r1, m->gate, m->up, nullptr, 0.f, m->hidden,
                                    inter, (int)B, act_mode)))
          return st;
      }
    }
    const void* w1[1] = {head.dev};
    float* y1[1] = {logits_dev};
    const int64_t r1[1] = {head.rows};
    return stream_fused_q8_0(ctx, 1, w1, y1, r1, m->hidden, nullptr, m->final_norm,
                             c.rms_norm_eps, nullptr, hidden, (int)B, act_mode);
  }

  for (uint32_t l = 0; l < c.num_hidden_layers; ++l) {
    auto& ly = m->layers[l];
    if (!ly.attn_norm || !ly.ffn_norm)
      return fail(ctx, KANSO_ERR_CONFIG, "decode_step: norm weights of layer %u not set", l);
    bool one = false;  // the launch below covered the whole group
    {
      const ModelLin* l3[3] = {&ly.w[KANSO_W_ATTN_Q], &ly.w[KANSO_W_ATTN_K], &ly.w[KANSO_W_ATTN_V]};
      float* y3[3] = {q, k, v};
      if ((st = lin_multi(ctx, 3, l3, y3, m->hidden, nullptr, ly.attn_norm, c.rms_norm_eps,
                          nullptr, B, act_mode, &one)))
        return st;
    }
    if (!one) {
      if ((st = launch_rmsnorm(ctx, m->hidden, ly.attn_norm, m->normed, B, hidden,
                               c.rms_norm_eps)))
        return st;
      if ((st = lin(ctx, ly.w[KANSO_W_ATTN_Q], m->normed, q, B, act_mode))) return st;
      if ((st = lin(ctx, ly.w[KANSO_W_ATTN_K], m->normed, k, B, act_mode))) return st;
      if ((st = lin(ctx, ly.w[KANSO_W_ATTN_V], m->normed, v, B, act_mode))) return st;
    }
    // The attention's merge also leaves its output as the packed f16 tile of the o-projection's
    // GEMM (when it can), which then starts without a pack launch of its own.
    const void* packed = nullptr;
    PaDecodeFusion fusion_l = fusion;
    if (act_mode == KANSO_ACT_F32) fusion_l.packed_out = &packed;
    if ((st = launch_paged_attention(ctx, kv, l, q, block_tables, context_lens, m->attn, &pa,
                                     max_ctx, &fusion_l)))
      return st;
    {
      const ModelLin* l1[1] = {&ly.w[KANSO_W_ATTN_OUTPUT]};
      float* y1[1] = {m->hidden};
      one = false;
      if (packed &&
          (st = lin_multi(ctx, 1, l1, y1, m->attn, nullptr, nullptr, 0.f, m->hidden, B, act_mode,
                          &one, packed)))
        return st;
      if (!one && (st = lin_multi(ctx, 1, l1, y1, m->attn, nullptr, nullptr, 0.f, m->hidden, B,
                                  act_mode, &one)))
        return st;
    }
    if (!one) {
      if ((st = lin(ctx, ly.w[KANSO_W_ATTN_OUTPUT], m->attn, m->proj, B, act_mode))) return st;
      if ((st = launch_residual_add(ctx, m->hidden, m->proj, (int64_t)B * hidden))) return st;
    }
    {
      const ModelLin* l2[2] = {&ly.w[KANSO_W_FFN_GATE], &ly.w[KANSO_W_FFN_UP]};
      float* y2[2] = {m->gate, m->up};
      if ((st = lin_multi(ctx, 2, l2, y2, m->hidden, nullptr, ly.ffn_norm, c.rms_norm_eps, nullptr,
                          B, act_mode, &one)))
        return st;
    }
    if (!one) {
      if ((st = launch_rmsnorm(ctx, m->hidden, ly.ffn_norm, m->normed, B, hidden, c.rms_norm_eps)))
        return st;
      if ((st = lin(ctx, ly.w[KANSO_W_FFN_GATE], m->normed, m->gate, B, act_mode))) return st;
      if ((st = lin(ctx, ly.w[KANSO_W_FFN_UP], m->normed, m->up, B, act_mode))) return st;
    }
    {
      const ModelLin* l1[1] = {&ly.w[KANSO_W_FFN_DOWN]};
      float* y1[1] = {m->hidden};
      if ((st = lin_multi(ctx, 1, l1, y1, m->gate, m->up, nullptr, 0.f, m->hidden, B, act_mode,
                          &one)))
        return st;
    }
    if (!one) {
      if ((st = launch_silu_mul(ctx, m->gate, m->up, m->act, (int64_t)B * inter))) return st;
      if ((st = lin(ctx, ly.w[KANSO_W_FFN_DOWN], m->act, m->proj, B, act_mode))) return st;
      if ((st = launch_residual_add(ctx, m->hidden, m->proj, (int64_t)B * hidden))) return st;
    }
  }
  {
    bool one = false;
    const ModelLin* l1[1] = {&head};
    float* y1[1] = {logits_dev};
    if ((st = lin_multi(ctx, 1, l1, y1, m->hidden, nullptr, m->final_norm, c.rms_norm_eps, nullptr,
                        B, act_mode, &one)) ||
        one)
      return st;
  }
  if ((st = launch_rmsnorm(ctx, m->hidden, m->final_norm, m->normed, B, hidden, c.rms_norm_eps)))
    return st;
  return lin(ctx, head, m->normed, logits_dev, B, act_mode);
}
