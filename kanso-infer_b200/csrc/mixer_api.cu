// Entry points to the single mechanisms of the latent attention, the matrix memory and the layers
// around them.
#include <algorithm>

#include "dense.cuh"

using namespace kanso;

namespace {
int32_t compute_of(const kanso_cuda_kv* kv) {
  return kv->kv_type == KANSO_KV_BF16 ? KANSO_COMPUTE_BF16 : KANSO_COMPUTE_F32;
}
RowMap row_map(const uint32_t* positions, const uint32_t* row_seq, const uint32_t* tables,
               uint32_t max_blocks) {
  RowMap m;
  m.positions = positions;
  m.row_seq = row_seq;
  m.tables = tables;
  m.max_blocks = max_blocks;
  return m;
}

// A call's own copies of host arrays on the device, freed when it ends.
struct CallMemory {
  kanso_cuda_ctx* ctx;
  std::vector<void*> mem;
  ~CallMemory() {
    cudaStreamSynchronize(ctx->stream);
    for (void* p : mem) cudaFree(p);
  }
  int32_t copy(const void* host, size_t bytes, void** out) {
    KANSO_CUDA_TRY(ctx, cudaMalloc(out, std::max<size_t>(bytes, 16)), "constants");
    mem.push_back(*out);
    if (host)
      KANSO_CUDA_TRY(ctx, cudaMemcpy(*out, host, bytes, cudaMemcpyHostToDevice), "constants");
    return KANSO_OK;
  }
};

int32_t latent_constants(kanso_cuda_ctx* ctx, const kanso_latent_attention_params* p,
                         CallMemory* mem, LatentAttn* a) {
  if (!p->num_heads || !p->dim || !p->rank || !p->rot || p->rot % 2 || !(p->rot_base > 0))
    return fail(ctx, KANSO_ERR_SHAPE, "latent attention: bad sizes");
  a->heads = p->num_heads;
  a->dim = p->dim;
  a->rot = p->rot;
  a->vdim = p->vdim;
  a->rank = p->rank;
  a->scale = p->scale;
  void *sink = nullptr, *freq = nullptr;
  const std::vector<double> f = rope_frequencies(p->rot, p->rot_base);
  int32_t st = mem->copy(f.data(), f.size() * sizeof(double), &freq);
  if (!st && p->sink) st = mem->copy(p->sink, (size_t)p->num_heads * 4, &sink);
  a->freq = (const double*)freq;
  a->sink = (const float*)sink;
  return st;
}
int32_t check_latent_pool(kanso_cuda_ctx* ctx, const kanso_cuda_kv* kv, uint32_t layer,
                          const kanso_latent_attention_params* p) {
  if (layer >= kv->dense.size() || kv->dense[layer].kv_heads != 1 ||
      kv->dense[layer].k_dim != p->rank + p->rot || kv->dense[layer].v_dim)
    return fail(ctx, KANSO_ERR_SHAPE, "latent attention: layer %u is not of %u + %u columns", layer,
                p->rank, p->rot);
  return KANSO_OK;
}
}  // namespace

extern "C" {

int32_t kanso_cuda_residual_norm(kanso_cuda_ctx* ctx, float* x, const float* y, const float* w,
                                 float eps, float mult, int32_t after_sum, int64_t T,
                                 int64_t width) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "residual_norm: ctx is NULL");
  if (!x || !y || !w || T < 0 || width < 1 || !aligned16(x) || !aligned16(y) || !aligned16(w))
    return fail(ctx, KANSO_ERR_SHAPE, "residual_norm: bad argument");
  if (!T) return KANSO_OK;
  ResidualSource r;
  r.y = y;
  return launch_residual_norm(ctx, KANSO_COMPUTE_F32, x, width, r, w, eps, mult,
                              after_sum ? Residual::kAddNorm : Residual::kAdd, nullptr, 0, T);
}

int32_t kanso_cuda_latent_store(kanso_cuda_ctx* ctx, kanso_cuda_kv* kv, uint32_t layer,
                                const float* down, uint32_t q_rank, const float* q_norm,
                                const float* c_norm, float eps, const uint32_t* positions,
                                const uint32_t* row_seq, const uint32_t* block_tables,
                                const kanso_latent_attention_params* p, void* cq) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "latent_store: ctx is NULL");
  if (!kv || !down || !q_rank || !q_norm || !c_norm || !positions || !block_tables || !p || !cq)
    return fail(ctx, KANSO_ERR_SHAPE, "latent_store: NULL argument");
  int32_t st = check_latent_pool(ctx, kv, layer, p);
  if (st || !p->num_rows) return st;
  CallMemory mem{ctx, {}};
  LatentStore s;
  if ((st = latent_constants(ctx, p, &mem, &s.a))) return st;
  s.down.d = down;
  s.down.ld = (int64_t)q_rank + p->rank + p->rot;
  s.down.q_rank = q_rank;
  s.down.q_norm = q_norm;
  s.down.c_norm = c_norm;
  s.down.eps = eps;
  s.kv = kv->dense[layer];
  s.map = row_map(positions, row_seq, block_tables, p->max_num_blocks_per_seq);
  s.status = ctx->dev_status;
  return launch_latent_down(ctx, compute_of(kv), s, cq, p->num_rows);
}

int32_t kanso_cuda_latent_attention(kanso_cuda_ctx* ctx, const kanso_cuda_kv* kv, uint32_t layer,
                                    const float* q_lat, const float* q, const uint32_t* positions,
                                    const uint32_t* row_seq, const uint32_t* block_tables,
                                    float* out, const kanso_latent_attention_params* p,
                                    int32_t path) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "latent_attention: ctx is NULL");
  if (!kv || !q_lat || !q || !positions || !block_tables || !out || !p || !p->sink)
    return fail(ctx, KANSO_ERR_SHAPE, "latent_attention: NULL argument");
  if (!aligned16(q_lat) || !aligned16(q) || !aligned16(out))
    return fail(ctx, KANSO_ERR_SHAPE, "latent_attention: arrays must be 16-byte aligned");
  int32_t st = check_latent_pool(ctx, kv, layer, p);
  if (st || !p->num_rows) return st;
  CallMemory mem{ctx, {}};
  LatentAttn a;
  if ((st = latent_constants(ctx, p, &mem, &a))) return st;
  LatentRows r;
  r.q_lat = q_lat;
  r.q_head = r.out_head = p->rank;
  r.q_row = r.out_row = (int64_t)p->num_heads * p->rank;
  r.q.q = q;
  r.q.ld = (int64_t)p->num_heads * (p->dim + p->rot);
  r.map = row_map(positions, row_seq, block_tables, p->max_num_blocks_per_seq);
  r.max_keys = p->max_num_blocks_per_seq * kv->dense[layer].block_size;
  r.out = out;
  r.out_f32 = true;
  r.n = p->num_rows;
  bool handled = false;
  st = launch_latent_attn_rows(ctx, compute_of(kv), a, kv->dense[layer], r, path, &handled);
  return st || handled ? st
                       : fail(ctx, KANSO_ERR_UNSUPPORTED, "latent_attention: sizes outside the "
                                                          "tile kernel");
}

int32_t kanso_cuda_softmax_prefill(kanso_cuda_ctx* ctx, const void* q, const void* q_rot,
                                   const void* k, const void* v, const void* k_rot, void* out,
                                   uint32_t pos0, const kanso_latent_attention_params* p) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "softmax_prefill: ctx is NULL");
  if (!q || !k || !v || !out || !p || (p->rot && (!q_rot || !k_rot)) || !p->num_heads)
    return fail(ctx, KANSO_ERR_SHAPE, "softmax_prefill: NULL argument");
  if (!aligned16(q) || !aligned16(q_rot) || !aligned16(k) || !aligned16(v) || !aligned16(k_rot) ||
      !aligned16(out))
    return fail(ctx, KANSO_ERR_SHAPE, "softmax_prefill: arrays must be 16-byte aligned");
  if (!p->num_rows) return KANSO_OK;
  std::vector<AttnTile> tiles;
  for (uint32_t r = 0; r < p->num_rows; r += 128)
    tiles.push_back({r, std::min(128u, p->num_rows - r), pos0 + r, 0});
  CallMemory mem{ctx, {}};
  void *dev = nullptr, *sink = nullptr;
  int32_t st = mem.copy(tiles.data(), tiles.size() * sizeof(AttnTile), &dev);
  if (!st && p->sink) st = mem.copy(p->sink, (size_t)p->num_heads * 4, &sink);
  if (st) return st;
  SoftmaxPrefill s;
  s.heads = p->num_heads;
  s.dim = p->dim;
  s.rot = p->rot;
  s.vdim = p->vdim;
  s.scale = p->scale;
  s.sink = (const float*)sink;
  s.q = (const bf16*)q;
  s.q_rot = (const bf16*)q_rot;
  s.q_rows = p->num_rows;
  s.k = (const bf16*)k;
  s.v = (const bf16*)v;
  s.k_rot = (const bf16*)k_rot;
  s.keys = (int64_t)pos0 + p->num_rows;
  s.k_ld = (int64_t)p->num_heads * round_up8(p->dim);
  s.v_ld = (int64_t)p->num_heads * round_up8(p->vdim);
  s.tiles = (const AttnTile*)dev;
  s.n_tiles = (uint32_t)tiles.size();
  s.out = (bf16*)out;
  s.out_ld = (int64_t)p->num_heads * p->vdim;
  bool handled = false;
  st = launch_softmax_prefill(ctx, s, &handled);
  return st || handled ? st
                       : fail(ctx, KANSO_ERR_UNSUPPORTED, "softmax_prefill: sizes outside the "
                                                          "kernel");
}

int32_t kanso_cuda_mlstm(kanso_cuda_ctx* ctx, kanso_cuda_kv* kv, uint32_t layer, const float* y,
                         const float* i_bias, const float* f_bias, float* out,
                         const kanso_mlstm_params* p, int32_t path) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "mlstm: ctx is NULL");
  if (!kv || !y || !i_bias || !f_bias || !out || !p)
    return fail(ctx, KANSO_ERR_SHAPE, "mlstm: NULL argument");
  if (!aligned16(y) || !aligned16(out))
    return fail(ctx, KANSO_ERR_SHAPE, "mlstm: arrays must be 16-byte aligned");
  if (layer >= kv->state.size() || !kv->state[layer].heads || p->slot >= kv->num_slots ||
      !(p->gate_cap > 0))
    return fail(ctx, KANSO_ERR_SHAPE, "mlstm: no state of layer %u in slot %u", layer, p->slot);
  if (!p->num_rows) return KANSO_OK;
  CallMemory mem{ctx, {}};
  const AttnTile portion = {0, p->num_rows, p->pos0, 0};
  void *dev = nullptr, *slot = nullptr, *work = nullptr;
  int32_t st = mem.copy(&portion, sizeof portion, &dev);
  if (!st) st = mem.copy(&p->slot, 4, &slot);
  if (st) return st;
  MlstmArgs a;
  a.state = kv->state[layer];
  a.heads = a.state.heads;
  a.dim = a.state.dim;
  a.vdim = a.state.vdim;
  a.cap = p->gate_cap;
  a.i_bias = i_bias;
  a.f_bias = f_bias;
  a.y = y;
  a.portions = (const AttnTile*)dev;
  a.slots = (const uint32_t*)slot;
  a.out = out;
  if (path == 1 || (path == 0 && p->num_rows < 16))
    return launch_mlstm_rows(ctx, a, 1, p->num_rows);
  if (!mlstm_chunk_fits(a))
    return path == 0 ? launch_mlstm_rows(ctx, a, 1, p->num_rows)
                     : fail(ctx, KANSO_ERR_UNSUPPORTED, "mlstm: heads of %u columns", a.dim);
  const size_t bytes = mlstm_chunk_bytes(a.heads, a.dim, a.vdim, p->num_rows);
  if ((st = mem.copy(nullptr, bytes, &work))) return st;
  return launch_mlstm_chunks(ctx, a, 1, p->num_rows, work, p->num_rows);
}

int32_t kanso_cuda_head_norm_gate(kanso_cuda_ctx* ctx, const float* o, const float* y,
                                  const float* w, float eps, float* out, int64_t T, uint32_t heads,
                                  uint32_t dim, uint32_t vdim) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "head_norm_gate: ctx is NULL");
  if (!o || !y || !w || !out || !heads || !dim || !vdim)
    return fail(ctx, KANSO_ERR_SHAPE, "head_norm_gate: bad argument");
  if (T < 1) return KANSO_OK;
  MlstmArgs a;
  a.heads = heads;
  a.dim = dim;
  a.vdim = vdim;
  a.y = y;
  a.out = const_cast<float*>(o);
  return launch_head_norm_gate(ctx, KANSO_COMPUTE_F32, a, w, eps, out, (int64_t)heads * vdim, T);
}

}  // extern "C"
