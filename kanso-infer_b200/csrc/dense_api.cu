// Entry points to the single mechanisms of the unquantised models.
#include <algorithm>

#include "dense.cuh"

using namespace kanso;

// The row-streaming kernels take f32 activations; this widens a bf16 x.
namespace {
__global__ void widen_kernel(const bf16* x, float* y, int64_t T, int64_t ld, int64_t cols) {
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < T * cols;
       i += (int64_t)gridDim.x * blockDim.x)
    y[i] = from_elem(x[i / cols * ld + i % cols]);
}
template <typename E>
__global__ void narrow_kernel(const float* x, E* y, int64_t T, int64_t ld, int64_t cols) {
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < T * ld;
       i += (int64_t)gridDim.x * blockDim.x)
    y[i] = to_elem<E>(i % ld < cols ? x[i / ld * cols + i % ld] : 0.f);
}
}  // namespace

static int32_t run_moe(kanso_cuda_ctx* ctx, int32_t compute, const float* x, const float* router,
                       const float* bias, RouteWeights form, const void* gate, const void* up,
                       const void* down, float* y, int64_t T, int64_t width, int64_t ff,
                       uint32_t experts, uint32_t top, int32_t path);

extern "C" {

int32_t kanso_cuda_sigmoid_attention(kanso_cuda_ctx* ctx, const kanso_cuda_kv* kv, uint32_t layer,
                                     const void* q, const uint32_t* positions,
                                     const uint32_t* row_seq, const uint32_t* block_tables,
                                     float* out, const kanso_sigmoid_attention_params* p,
                                     int32_t path) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "sigmoid_attention: ctx is NULL");
  if (!kv || !p || !q || !positions || !block_tables || !out)
    return fail(ctx, KANSO_ERR_SHAPE, "sigmoid_attention: NULL argument");
  if (!aligned16(q) || !aligned16(out))
    return fail(ctx, KANSO_ERR_SHAPE, "sigmoid_attention: q and out must be 16-byte aligned");
  if (layer >= kv->dense.size())
    return fail(ctx, KANSO_ERR_SHAPE, "sigmoid_attention: no unquantised layer %u", layer);
  const KvDenseLayer& d = kv->dense[layer];
  if (!p->num_heads || p->num_heads % d.kv_heads)
    return fail(ctx, KANSO_ERR_SHAPE, "sigmoid_attention: %u heads over %u key/value heads",
                p->num_heads, d.kv_heads);
  if (!p->num_rows) return KANSO_OK;
  const int32_t compute = kv->kv_type == KANSO_KV_BF16 ? KANSO_COMPUTE_BF16 : KANSO_COMPUTE_F32;
  SigmoidAttn a;
  void* mem = nullptr;
  int32_t st = make_sigmoid_attn(ctx, p->num_heads, p->window, p->scale, p->softcap, p->r1, p->r2,
                                 p->pb, &a, &mem);
  RowMap map;
  map.positions = positions;
  map.row_seq = row_seq;
  map.tables = block_tables;
  map.max_blocks = p->max_num_blocks_per_seq;
  const int64_t out_ld = (int64_t)p->num_heads * d.v_dim;
  AttnTile* dev = nullptr;
  bool handled = false;
  if (!st && path >= 2) {
    const uint32_t step = path == 3 ? 128 : 64;
    std::vector<uint32_t> pos(p->num_rows), seq(p->num_rows, 0);
    cudaError_t e = cudaStreamSynchronize(ctx->stream);
    if (e == cudaSuccess)
      e = cudaMemcpy(pos.data(), positions, pos.size() * 4, cudaMemcpyDeviceToHost);
    if (e == cudaSuccess && row_seq)
      e = cudaMemcpy(seq.data(), row_seq, seq.size() * 4, cudaMemcpyDeviceToHost);
    std::vector<AttnTile> tiles;
    for (uint32_t r = 0; r < p->num_rows; r += step) {
      tiles.push_back({r, std::min(step, p->num_rows - r), pos[r], seq[0]});
      for (uint32_t k = r; k < std::min(r + step, p->num_rows); ++k)
        if (pos[k] != pos[r] + (k - r) || seq[k] != seq[0])
          st = fail(ctx, KANSO_ERR_SHAPE, "sigmoid_attention: the tile kernel needs one sequence's "
                                          "consecutive positions");
    }
    if (e == cudaSuccess) e = cudaMalloc((void**)&dev, tiles.size() * sizeof(AttnTile));
    if (e == cudaSuccess)
      e = cudaMemcpy(dev, tiles.data(), tiles.size() * sizeof(AttnTile), cudaMemcpyHostToDevice);
    if (!st && e != cudaSuccess) st = cuda_fail(ctx, e, "sigmoid_attention");
    if (!st && compute == KANSO_COMPUTE_BF16 && path == 3)
      st = launch_sigmoid_attn_prefill(ctx, a, d, q, p->num_rows, map, dev, (uint32_t)tiles.size(),
                                       out, true, out_ld, &handled);
    else if (!st && compute == KANSO_COMPUTE_BF16)
      st = launch_sigmoid_attn_tiles(ctx, a, d, q, map, dev, (uint32_t)tiles.size(), out, true,
                                     out_ld, &handled);
    if (!st && !handled)
      st = fail(ctx, KANSO_ERR_UNSUPPORTED, "sigmoid_attention: sizes outside the tile kernel");
  } else if (!st) {
    const uint32_t max_keys = p->max_num_blocks_per_seq * d.block_size;
    st = launch_sigmoid_attn_rows(ctx, compute, a, d, q, nullptr, map, max_keys, out, true, out_ld,
                                  p->num_rows);
  }
  cudaStreamSynchronize(ctx->stream);  // the constants are this call's own
  if (mem) cudaFree(mem);
  if (dev) cudaFree(dev);
  return st;
}

int32_t kanso_cuda_qk_norm_store(kanso_cuda_ctx* ctx, kanso_cuda_kv* kv, uint32_t layer,
                                 const float* qkv, const float* q_norm, const float* k_norm,
                                 float eps, uint32_t num_heads, const uint32_t* positions,
                                 const uint32_t* row_seq, const uint32_t* block_tables,
                                 uint32_t max_blocks, uint32_t T, void* q_out) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "qk_norm_store: ctx is NULL");
  if (!kv || !qkv || !q_norm || !k_norm || !positions || !block_tables || !q_out)
    return fail(ctx, KANSO_ERR_SHAPE, "qk_norm_store: NULL argument");
  if (!aligned16(qkv) || !aligned16(q_norm) || !aligned16(k_norm) || !aligned16(q_out))
    return fail(ctx, KANSO_ERR_SHAPE, "qk_norm_store: arrays must be 16-byte aligned");
  if (layer >= kv->dense.size())
    return fail(ctx, KANSO_ERR_SHAPE, "qk_norm_store: no unquantised layer %u", layer);
  if (!T) return KANSO_OK;
  QkvSource s;
  s.qkv = qkv;
  s.q_norm = q_norm;
  s.k_norm = k_norm;
  s.eps = eps;
  RowMap map;
  map.positions = positions;
  map.row_seq = row_seq;
  map.tables = block_tables;
  map.max_blocks = max_blocks;
  return launch_qk_norm_store(ctx,
                              kv->kv_type == KANSO_KV_BF16 ? KANSO_COMPUTE_BF16 : KANSO_COMPUTE_F32,
                              s, kv->dense[layer], num_heads, map, q_out, T);
}

int32_t kanso_cuda_dense_linear(kanso_cuda_ctx* ctx, int32_t compute, const void* w,
                                const void* x, float* y, int64_t T, int64_t rows, int64_t cols,
                                int32_t path) {
  return kanso_cuda_dense_linear_act(ctx, compute, w, x, nullptr, 0, y, T, rows, cols, path);
}

int32_t kanso_cuda_dense_linear_act(kanso_cuda_ctx* ctx, int32_t compute, const void* w,
                                    const void* x, const float* bias, int32_t relu2, float* y,
                                    int64_t T, int64_t rows, int64_t cols, int32_t path) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "dense_linear: ctx is NULL");
  if (!w || !x || !y || T < 0 || rows < 1 || cols < 1)
    return fail(ctx, KANSO_ERR_SHAPE, "dense_linear: bad argument");
  if (!aligned16(w) || !aligned16(x) || !aligned16(y))
    return fail(ctx, KANSO_ERR_SHAPE, "dense_linear: arrays must be 16-byte aligned");
  if (T == 0) return KANSO_OK;
  DenseMat m;
  m.w = const_cast<void*>(w);
  m.rows = rows;
  m.cols = cols;
  m.ld = round_up8(cols);
  if (path == 1 || (path == 0 && T <= GEMV_MAX_T)) {
    GemvSource g;
    if (compute == KANSO_COMPUTE_BF16) {
      int32_t st = ctx_stage_dev(ctx, (size_t)(T * cols) * 4);
      if (st) return st;
      widen_kernel<<<256, 256, 0, ctx->stream>>>((const bf16*)x, (float*)ctx->stage_dev, T, m.ld,
                                                 cols);
      if ((st = after_launch(ctx, "widen"))) return st;
      g.x = (const float*)ctx->stage_dev;
    } else {
      if (m.ld != cols)
        return fail(ctx, KANSO_ERR_UNSUPPORTED, "dense_linear: row streaming of padded f32 rows");
      g.x = (const float*)x;
    }
    GemvOut o;
    o.bias = bias;
    o.relu2 = relu2 != 0;
    return launch_gemv(ctx, compute, m, g, y, rows, (int)T, o);
  }
  GemmRows r;
  r.T = T;
  GemmOut o;
  o.bias = bias;
  o.relu2 = relu2 != 0;
  int splits = 1;
  return launch_gemm(ctx, compute, m, x, y, rows, r, 1, &splits, 0, o);
}

int32_t kanso_cuda_moe(kanso_cuda_ctx* ctx, int32_t compute, const float* x, const float* router,
                       const void* gate, const void* up, const void* down, float* y, int64_t T,
                       int64_t width, int64_t ff, uint32_t experts, uint32_t top, int32_t path) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "moe: ctx is NULL");
  if (!gate || !aligned16(gate)) return fail(ctx, KANSO_ERR_SHAPE, "moe: bad argument");
  return run_moe(ctx, compute, x, router, nullptr, RouteWeights::kShares, gate, up, down, y, T,
                 width, ff, experts, top, path);
}

int32_t kanso_cuda_moe_relu2(kanso_cuda_ctx* ctx, int32_t compute, const float* x,
                             const float* router, const float* router_bias, const void* up,
                             const void* down, float* y, int64_t T, int64_t width, int64_t ff,
                             uint32_t experts, uint32_t top, int32_t path) {
  if (!ctx) return fail(nullptr, KANSO_ERR_CONFIG, "moe: ctx is NULL");
  return run_moe(ctx, compute, x, router, router_bias, RouteWeights::kChosenSoftmax, nullptr, up,
                 down, y, T, width, ff, experts, top, path);
}

}  // extern "C"

// gate nullptr: experts of max(0, up x)^2
static int32_t run_moe(kanso_cuda_ctx* ctx, int32_t compute, const float* x, const float* router,
                       const float* bias, RouteWeights form, const void* gate, const void* up,
                       const void* down, float* y, int64_t T, int64_t width, int64_t ff,
                       uint32_t experts, uint32_t top, int32_t path) {
  if (!x || !router || !up || !down || !y || T < 0 || width < 1 || ff < 1 || !experts || !top ||
      top > experts)
    return fail(ctx, KANSO_ERR_SHAPE, "moe: bad argument");
  if (!aligned16(x) || !aligned16(router) || !aligned16(up) || !aligned16(down) || !aligned16(y))
    return fail(ctx, KANSO_ERR_SHAPE, "moe: arrays must be 16-byte aligned");
  if (T == 0) return KANSO_OK;
  auto mat = [&](const void* w, int64_t rows, int64_t cols, int64_t groups) {
    DenseMat m;
    m.w = const_cast<void*>(w);
    m.rows = rows;
    m.cols = cols;
    m.ld = round_up8(cols);
    m.groups = groups;
    return m;
  };
  const DenseMat r = mat(router, experts, width, 1), g = mat(gate, ff, width, experts),
                 u = mat(up, ff, width, experts), d = mat(down, width, ff, experts);
  const int64_t WL = g.ld, FL = d.ld, R = T * top;
  const size_t es = compute == KANSO_COMPUTE_BF16 ? 2 : 4;
  // one allocation of the call's own
  uint8_t* mem = nullptr;
  size_t total = 0;
  auto room = [&](size_t bytes) {
    const size_t at = total;
    total += (bytes + 255) & ~(size_t)255;
    return at;
  };
  const size_t o_rl = room((size_t)(T * experts) * 4), o_sel = room((size_t)R * 4),
               o_w = room((size_t)R * 4), o_slot = room((size_t)R * 4),
               o_cnt = room((size_t)experts * 4), o_off = room((size_t)(experts + 1) * 4),
               o_a32 = room((size_t)(R * FL) * 4), o_xe = room((size_t)(T * WL) * es),
               o_xs = room((size_t)(R * WL) * es), o_act = room((size_t)(R * FL) * es),
               o_ye = room((size_t)(R * width) * 4);
  KANSO_CUDA_TRY(ctx, cudaMalloc((void**)&mem, total), "moe");
  cudaMemsetAsync(mem, 0, total, ctx->stream);
  float *rl = (float*)(mem + o_rl), *wgt = (float*)(mem + o_w), *a32 = (float*)(mem + o_a32),
        *ye = (float*)(mem + o_ye);
  uint32_t *sel = (uint32_t*)(mem + o_sel), *slot = (uint32_t*)(mem + o_slot),
           *cnt = (uint32_t*)(mem + o_cnt), *off = (uint32_t*)(mem + o_off);
  int32_t st = KANSO_OK;
  if (path == 1 || (path == 0 && T <= GEMV_MAX_T)) {
    GemvSource src;
    src.x = x;
    GemvOut o;
    o.bias = bias;
    st = launch_gemv(ctx, KANSO_COMPUTE_F32, r, src, rl, experts, (int)T, o);
    if (!st)
      st = launch_gemv_gate_up(ctx, compute, gate ? &g : nullptr, u, x, rl, experts, top, form, a32,
                               sel, (int)T);
    if (!st) st = launch_gemv_down(ctx, compute, d, a32, sel, top, y, (int)T);
  } else {
    if (compute == KANSO_COMPUTE_BF16)
      narrow_kernel<bf16><<<256, 256, 0, ctx->stream>>>(x, (bf16*)(mem + o_xe), T, WL, width);
    else
      narrow_kernel<float><<<256, 256, 0, ctx->stream>>>(x, (float*)(mem + o_xe), T, WL, width);
    st = after_launch(ctx, "narrow");
    if (!st) st = launch_route(ctx, x, width, r, bias, top, form, sel, wgt, cnt, slot, T);
    if (!st)
      st = launch_expert_gather(ctx, compute, cnt, experts, top, sel, slot, off, mem + o_xe, WL,
                                mem + o_xs, T);
    GemmRows er;
    er.T = R;
    er.offsets = off;
    er.groups = (int)experts;
    int splits = 1;
    GemmOut act;
    act.elem = act.relu2 = true;
    if (!st)
      st = gate ? launch_gemm_gate_up(ctx, compute, g, u, mem + o_xs, mem + o_act, FL, er)
                : launch_gemm(ctx, compute, u, mem + o_xs, mem + o_act, FL, er, 1, &splits, 0, act);
    if (!st) st = launch_gemm(ctx, compute, d, mem + o_act, ye, width, er, 1, &splits, 0);
    if (!st) st = launch_expert_sum(ctx, ye, slot, wgt, top, y, width, T);
  }
  cudaStreamSynchronize(ctx->stream);
  cudaFree(mem);
  return st;
}
