// Unquantised (bfloat16 or f32) layers: what the row-streaming kernels, the tile kernels, the
// expert routing, the attentions and the recurrence share, and their launchers.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>

#include <vector>

#include "glue.cuh"
#include "kv_pool.h"

namespace kanso {

using bf16 = __nv_bfloat16;

inline uint32_t round_up8(int64_t n) { return (uint32_t)((n + 7) & ~(int64_t)7); }

// ---- eight consecutive elements (16-byte aligned) to and from f32 ----
__device__ __forceinline__ void unpack_bf16x2(uint32_t u, float& lo, float& hi) {
  lo = __uint_as_float(u << 16);
  hi = __uint_as_float(u & 0xFFFF0000u);
}
struct Raw8b {
  uint4 a;
};
struct Raw8f {
  float4 a, b;
};
__device__ __forceinline__ Raw8b load_raw(const bf16* p) {
  return {*reinterpret_cast<const uint4*>(p)};
}
__device__ __forceinline__ Raw8f load_raw(const float* p) {
  return {*reinterpret_cast<const float4*>(p), *reinterpret_cast<const float4*>(p + 4)};
}
// the same through the streaming path: weights are read once per launch
__device__ __forceinline__ Raw8b load_raw_once(const bf16* p) {
  Raw8b r;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(r.a.x), "=r"(r.a.y), "=r"(r.a.z), "=r"(r.a.w)
               : "l"(p));
  return r;
}
__device__ __forceinline__ Raw8f load_raw_once(const float* p) {
  return {__ldcs(reinterpret_cast<const float4*>(p)), __ldcs(reinterpret_cast<const float4*>(p + 4))};
}
__device__ __forceinline__ void expand(const Raw8b& r, float (&v)[8]) {
  unpack_bf16x2(r.a.x, v[0], v[1]);
  unpack_bf16x2(r.a.y, v[2], v[3]);
  unpack_bf16x2(r.a.z, v[4], v[5]);
  unpack_bf16x2(r.a.w, v[6], v[7]);
}
__device__ __forceinline__ void expand(const Raw8f& r, float (&v)[8]) {
  v[0] = r.a.x, v[1] = r.a.y, v[2] = r.a.z, v[3] = r.a.w;
  v[4] = r.b.x, v[5] = r.b.y, v[6] = r.b.z, v[7] = r.b.w;
}
template <typename E>
__device__ __forceinline__ E to_elem(float v);
template <>
__device__ __forceinline__ bf16 to_elem<bf16>(float v) {
  return __float2bfloat16_rn(v);
}
template <>
__device__ __forceinline__ float to_elem<float>(float v) {
  return v;
}
__device__ __forceinline__ float from_elem(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float from_elem(float v) { return v; }

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float relu_squared(float z) {
  const float r = fmaxf(z, 0.f);
  return r * r;
}

// How the weights of the chosen experts come about: as their shares of the softmax over all
// experts, or as the softmax over the chosen ones alone.
enum class RouteWeights : int { kShares, kChosenSoftmax };

// The `top` largest of the router's logits in `l` (shared memory, overwritten), ties to the lower
// number, and their weights. One warp.
__device__ __forceinline__ void warp_route(float* l, int experts, int top, RouteWeights form,
                                           int lane, uint32_t* sel, float* weight) {
  float m = -INFINITY;
  for (int e = lane; e < experts; e += 32) m = fmaxf(m, l[e]);
#pragma unroll
  for (int o = 16; o; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, o));
  float sum = 0.f;
  for (int e = lane; e < experts; e += 32) sum += expf(l[e] - m);
#pragma unroll
  for (int o = 16; o; o >>= 1) sum += __shfl_xor_sync(0xFFFFFFFFu, sum, o);
  float chosen = 0.f;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
    int at = experts;
    for (int e = lane; e < experts; e += 32)
      if (l[e] > best) {
        best = l[e];
        at = e;
      }
#pragma unroll
    for (int o = 16; o; o >>= 1) {
      const float v = __shfl_xor_sync(0xFFFFFFFFu, best, o);
      const int i = __shfl_xor_sync(0xFFFFFFFFu, at, o);
      if (v > best || (v == best && i < at)) {
        best = v;
        at = i;
      }
    }
    if (at >= experts) at = j;  // no finite logit is left
    const float e = expf(best - m);
    chosen += e;
    if (lane == 0) {
      sel[j] = (uint32_t)at;
      weight[j] = form == RouteWeights::kShares ? e / sum : e;
      l[at] = -INFINITY;
    }
    __syncwarp();
  }
  if (form == RouteWeights::kChosenSoftmax)
    for (int j = lane; j < top; j += 32) weight[j] /= chosen;
  __syncwarp();
}

// A weight matrix [groups][rows][ld] on the device, ld = cols rounded up to 8, zeros behind.
struct DenseMat {
  void* w = nullptr;
  int64_t rows = 0, cols = 0, ld = 0, groups = 1;
};

// Where a row of the step lies: its position and the block table of its sequence.
struct RowMap {
  const uint32_t* positions = nullptr;
  const uint32_t* row_seq = nullptr;  // nullptr: row t belongs to sequence t
  const uint32_t* tables = nullptr;
  uint32_t max_blocks = 0;
};

// ---- row streaming: few activation rows (csrc/gemv_dense.cu) ----
// How the activations of a launch come about; every CTA repeats it. With y, the residual step that
// belongs in front of the product (y = the sum of `parts` partial results), which one CTA writes
// to x_out:
//   x' = x + mult * rmsnorm(y) * norm_w            kAdd
//   x' = rmsnorm(mult * x + y) * norm_w            kAddNorm
// With final_w a second norm of x' is what enters the product. x and x_out must differ. Without
// y, `gate` makes the product's input from heads: each head of x (cols / heads columns) over its
// own root mean square, times norm_w, times sigmoid(gate).
enum class Residual : int { kAdd, kAddNorm };
struct GemvSource {
  const float* x = nullptr;
  // Rows of x that lie further apart than the columns (not 0; without y), and from one weight
  // group's input to the next's.
  int64_t x_ld = 0, x_group = 0;
  float* x_out = nullptr;
  const float* y = nullptr;
  int parts = 1;
  int64_t part_stride = 0;
  const float* norm_w = nullptr;
  const float* final_w = nullptr;
  float eps = 0.f, mult = 0.f;
  Residual form = Residual::kAdd;
  const float* gate = nullptr;
  int64_t gate_ld = 0;
  int heads = 0;
  const uint32_t* row_index = nullptr;  // row of the launch -> row of x and y
};
// What becomes of a product's results on the way out.
struct GemvOut {
  const float* bias = nullptr;  // [rows]
  bool relu2 = false;           // max(0, z)^2
  int64_t group_step = 0;       // from one weight group's results to the next's
};
constexpr int64_t GEMV_MAX_COLS = 50 * 1024;  // columns of a row in shared memory
constexpr int GEMV_MAX_T = 2;  // more rows: the tile kernels are faster
struct LatentStore;
// out[T][rows] = source @ W^T (f32 out), group by group where W has several. `store`: work on the
// step's own cache rows that one more CTA does beside the product (see LatentStore).
int32_t launch_gemv(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat& w, const GemvSource& s,
                    float* out, int64_t out_ld, int T, const GemvOut& o = GemvOut(),
                    const LatentStore* store = nullptr);
// Experts of the chosen rows: act[T*top][ff ld] = weight * silu(gate x) * (up x), without a gate
// weight * max(0, up x)^2; the weight and the choice are taken from the router's logits;
// sel[T*top] receives the expert numbers.
int32_t launch_gemv_gate_up(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat* gate,
                            const DenseMat& up, const float* x, const float* router_logits,
                            uint32_t experts, uint32_t top, RouteWeights form, float* act,
                            uint32_t* sel, int T);
// out[T][rows] = sum over the top experts of W_sel act
int32_t launch_gemv_down(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat& down,
                         const float* act, const uint32_t* sel, uint32_t top, float* out, int T);

// ---- tiles: many activation rows (csrc/gemm_dense.cu) ----
// Rows of the activations and of the result are grouped: rows [offsets[g], offsets[g+1]) use
// weight group g; offsets nullptr: `groups` groups of T / groups rows.
struct GemmRows {
  int64_t T = 0;
  const uint32_t* offsets = nullptr;
  int groups = 1;
};
// What becomes of a product's results on the way out.
struct GemmOut {
  const float* bias = nullptr;  // [rows], the same for every group
  bool relu2 = false;           // max(0, z)^2 (not with a split)
  bool elem = false;            // results in the products' element type, pad columns zero
  // Not 0 (equal groups only): row r of group g lies at r * y_ld + g * group_step instead of behind
  // the groups before it.
  int64_t group_step = 0;
  const uint32_t* rows = nullptr;  // with group_step: row r of a group goes to row rows[r]
};
// y[T][rows] = x[T][ld] W^T, f32 unless `o` says otherwise. With *splits > 1 on return the result
// is the sum of that many arrays [T][y_ld], `part_stride` elements apart (only when max_splits
// allows it).
int32_t launch_gemm(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat& w, const void* x, void* y,
                    int64_t y_ld, const GemmRows& r, int max_splits, int* splits,
                    int64_t part_stride, const GemmOut& o = GemmOut());
// act[T][act_ld] = silu(x W_gate^T) * (x W_up^T), element type by compute, pad columns zero
int32_t launch_gemm_gate_up(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat& gate,
                            const DenseMat& up, const void* x, void* act, int64_t act_ld,
                            const GemmRows& r);

// ---- norms and expert routing on many rows (csrc/dense_rows.cu) ----
// x[t] = embed[token] * scale, and the same as the products' element type in xe [T][ld]
int32_t launch_embed_scaled(kanso_cuda_ctx* ctx, int32_t compute, const void* embed, int64_t ld,
                            const uint32_t* tokens, int64_t vocab, float scale, float* x,
                            int64_t width, void* xe, int64_t T);
// Source of the value that the residual step normalises.
struct ResidualSource {
  const float* y = nullptr;  // [parts][T][width] or, with slot, expert outputs [T*top][width]
  int parts = 1;
  int64_t part_stride = 0;
  const uint32_t* slot = nullptr;  // [T*top]: where the output of a (row, choice) pair lies
  const float* weight = nullptr;   // [T*top]
  int top = 0;
};
// y[t] = the weighted sum of a row's expert outputs, without the residual step
int32_t launch_expert_sum(kanso_cuda_ctx* ctx, const float* ye, const uint32_t* slot,
                          const float* weight, uint32_t top, float* y, int64_t width, int64_t T);
// The residual step in place (see Residual); xe as above (nullptr: not wanted)
int32_t launch_residual_norm(kanso_cuda_ctx* ctx, int32_t compute, float* x, int64_t width,
                             const ResidualSource& s, const float* w, float eps, float mult,
                             Residual form, void* xe, int64_t xe_ld, int64_t T);
// out[i] = rmsnorm(x[rows[i]]) * w as the products' element type
int32_t launch_norm_rows(kanso_cuda_ctx* ctx, int32_t compute, const float* x, int64_t width,
                         const uint32_t* rows, const float* w, float eps, void* out,
                         int64_t out_ld, int64_t n);
// RMS norm over the whole q row and the whole k row of qkv, then q to q_out, k and v to the pool
struct QkvSource {
  const float* qkv = nullptr;  // [parts][T][H*k_dim + G*k_dim + G*v_dim]
  int parts = 1;
  int64_t part_stride = 0;
  const float* q_norm = nullptr;
  const float* k_norm = nullptr;
  float eps = 0.f;
};
int32_t launch_qk_norm_store(kanso_cuda_ctx* ctx, int32_t compute, const QkvSource& s,
                             const KvDenseLayer& kv, uint32_t H, const RowMap& map, void* q_out,
                             int64_t T);
// Router (f32 weights, bias or nullptr) and choice: the experts and their weights per (row, place),
// rows per expert in counts (cleared by the caller), place within the expert in slot
int32_t launch_route(kanso_cuda_ctx* ctx, const float* x, int64_t width, const DenseMat& router,
                     const float* bias, uint32_t top, RouteWeights form, uint32_t* sel, float* weight, uint32_t* counts, uint32_t* slot,
                     int64_t T);
// offsets[experts + 1] from counts; slot becomes the row of the sorted order; xs = rows of xe
// in that order
int32_t launch_expert_gather(kanso_cuda_ctx* ctx, int32_t compute, const uint32_t* counts,
                             uint32_t experts, uint32_t top, const uint32_t* sel, uint32_t* slot,
                             uint32_t* offsets, const void* xe, int64_t ld, void* xs, int64_t T);

// ---- sigmoid attention (csrc/sigmoid_attention.cu) ----
// Constants of one layer. bias holds pb[h] - r1[h] ln(1 + r2[h] d) for d < bias_len.
struct SigmoidAttn {
  uint32_t heads = 0, window = 0;
  float scale = 1.f, softcap = 0.f;
  const float* bias = nullptr;
  uint32_t bias_len = 0;
  const float* r1 = nullptr;  // device, for distances beyond bias_len
  const float* r2 = nullptr;
  const float* pb = nullptr;
};
constexpr uint32_t ATTN_BIAS_MAX = 8192;
// A tile of consecutive rows of one sequence.
struct AttnTile {
  uint32_t row0, rows, pos0, seq;
};
// Uploads r1, r2, pb and the table; `mem` receives one allocation to free.
int32_t make_sigmoid_attn(kanso_cuda_ctx* ctx, uint32_t heads, uint32_t window, float scale,
                          float softcap, const float* r1, const float* r2, const float* pb,
                          SigmoidAttn* out, void** mem);
// One CTA per (share of the keys, kv head, row). `fused`: the rows' own q, k, v come raw from
// there, are normalised here, and k and v are stored to the pool by the CTA that reads the last
// key; every row must then be its sequence's only one in the step. Otherwise q is given.
// out_f32: out is f32, else the products' element type. max_keys bounds a row's visible keys.
int32_t launch_sigmoid_attn_rows(kanso_cuda_ctx* ctx, int32_t compute, const SigmoidAttn& a,
                                 const KvDenseLayer& kv, const void* q, const QkvSource* fused,
                                 const RowMap& map, uint32_t max_keys, void* out, bool out_f32,
                                 int64_t out_ld, int64_t T);
// bf16 prompts on tcgen05, tiles of up to 128 rows (csrc/sigmoid_prefill.cu); q has q_rows rows.
// *handled = false when a size is outside the kernel's range (no window, a window beyond the table,
// heads beyond 256, other pages than 8, 16, 32 or 64 tokens).
int32_t launch_sigmoid_attn_prefill(kanso_cuda_ctx* ctx, const SigmoidAttn& a,
                                    const KvDenseLayer& kv, const void* q, int64_t q_rows,
                                    const RowMap& map, const AttnTile* tiles, uint32_t n_tiles,
                                    void* out, bool out_f32, int64_t out_ld, bool* handled);
// bf16 mma.sync tiles of up to 64 rows; *handled = false when a size is outside the kernel's range.
int32_t launch_sigmoid_attn_tiles(kanso_cuda_ctx* ctx, const SigmoidAttn& a,
                                  const KvDenseLayer& kv, const void* q, const RowMap& map,
                                  const AttnTile* tiles, uint32_t n_tiles, void* out,
                                  bool out_f32, int64_t out_ld, bool* handled);

// ---- rotation (csrc/dense_rows.cu) ----
// The angle position * freq in f64, brought into one turn before it becomes f32: far positions keep
// the whole accuracy of the sine and cosine.
__device__ __forceinline__ void rope_sincos(uint32_t position, double freq, float* s, float* c) {
  const double turn = 6.283185307179586476925287;
  const double a = (double)position * freq;
  sincosf((float)(a - turn * rint(a / turn)), s, c);
}
// freq[i] = base^(-2i / dims), i < dims / 2; the pair (2i, 2i + 1) turns by position * freq[i].
std::vector<double> rope_frequencies(uint32_t dims, double base);

// ---- latent attention (csrc/latent_attention.cu, csrc/softmax_prefill.cu, csrc/dense_rows.cu) ----
// Softmax attention whose keys and values are linear in a latent c of `rank` columns that all heads
// share; a token's cache row is [c | rotated key part of `rot` columns] (KvDenseLayer with one
// head, k_dim = rank + rot, no values). The denominator also holds exp(sink[h]).
struct LatentAttn {
  uint32_t heads = 0, dim = 0, rot = 0, vdim = 0, rank = 0;
  float scale = 1.f;
  const float* sink = nullptr;   // device [heads]
  const double* freq = nullptr;  // device [rot / 2]
};
// A row's down projection [query latent (q_rank) | c (rank) | key part (rot)], f32, as the sum of
// parts; norm weights of the first two.
struct LatentDown {
  const float* d = nullptr;
  int parts = 1;
  int64_t part_stride = 0;
  int64_t ld = 0;
  uint32_t q_rank = 0;
  const float* q_norm = nullptr;
  const float* c_norm = nullptr;
  float eps = 0.f;
};
// The cache rows of the step's tokens from their down projections: norm of c, rotation of the key
// part, store.
struct LatentStore {
  LatentAttn a;
  LatentDown down;
  KvDenseLayer kv;
  RowMap map;
  int* status = nullptr;
};
// Sine and cosine of the thread's first pair of columns: nothing in front is needed for them.
__device__ __forceinline__ float2 latent_turn(const LatentStore& s, int64_t t) {
  float2 r = make_float2(0.f, 1.f);
  if (threadIdx.x < s.a.rot / 2)
    rope_sincos(s.map.positions[t], s.a.freq[threadIdx.x], &r.x, &r.y);
  return r;
}
template <typename E>
__device__ __forceinline__ void latent_store_row(const LatentStore& s, int64_t t, float2 turn,
                                                 float* red) {
  const LatentDown& p = s.down;
  const float* src = p.d + t * p.ld + p.q_rank;
  auto value = [&](int i) {
    float v = src[i];
#pragma unroll 3
    for (int k = 1; k < p.parts; ++k) v += src[k * p.part_stride + i];
    return v;
  };
  const KvDenseLayer& kv = s.kv;
  const int R = s.a.rank, RD = s.a.rot;
  const uint32_t pos = s.map.positions[t];
  const uint32_t seq = s.map.row_seq ? s.map.row_seq[t] : (uint32_t)t;
  const uint32_t place = pos / kv.block_size;
  uint32_t block = kv.num_blocks;
  if (place < s.map.max_blocks) block = s.map.tables[(int64_t)seq * s.map.max_blocks + place];
  constexpr int KEEP = 4;  // values a thread keeps between the two passes
  float kept[KEEP], ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    kept[k] = i < R ? value(i) : 0.f;
    ss += kept[k] * kept[k];
  }
  for (int i = threadIdx.x + KEEP * blockDim.x; i < R; i += blockDim.x) {
    const float v = value(i);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  if (block >= kv.num_blocks) {
    if (threadIdx.x == 0) atomicOr(s.status, DEV_BAD_INDEX);
    return;
  }
  const float inv = 1.0f / sqrtf(ss / (float)R + p.eps);
  E* dst = reinterpret_cast<E*>(kv.base) + kv.k_elem(block, 0, pos % kv.block_size);
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < R) dst[i] = to_elem<E>(kept[k] * inv * p.c_norm[i]);
  }
  for (int i = threadIdx.x + KEEP * blockDim.x; i < R; i += blockDim.x)
    dst[i] = to_elem<E>(value(i) * inv * p.c_norm[i]);
  for (int i = threadIdx.x; i < RD / 2; i += blockDim.x) {
    if (i != threadIdx.x) rope_sincos(pos, s.a.freq[i], &turn.x, &turn.y);
    const float u = value(R + 2 * i), v = value(R + 2 * i + 1);
    dst[R + 2 * i] = to_elem<E>(u * turn.y - v * turn.x);
    dst[R + 2 * i + 1] = to_elem<E>(v * turn.y + u * turn.x);
  }
}
// The store, and the normed query latents cq [T][q_rank ld] in the products' element type.
int32_t launch_latent_down(kanso_cuda_ctx* ctx, int32_t compute, const LatentStore& s, void* cq,
                           int64_t T);
// Queries of the step's rows, f32 as the sum of parts, row t's head h at t * ld + h * (dim + rot).
struct LatentQuery {
  const float* q = nullptr;
  int parts = 1;
  int64_t part_stride = 0;
  int64_t ld = 0;
};
// The unrotated parts of the listed rows (nullptr: all), head by head: out [heads][n][dim ld]
int32_t launch_latent_q_heads(kanso_cuda_ctx* ctx, int32_t compute, const LatentAttn& a,
                              const LatentQuery& q, const uint32_t* rows, int64_t n, void* out);
// bf16 queries of all rows: q [T][heads][dim ld] and the rotated parts q_rot [T][heads][rot ld]
int32_t launch_latent_q_rows(kanso_cuda_ctx* ctx, const LatentAttn& a, const LatentQuery& q,
                             const uint32_t* positions, bf16* out, bf16* out_rot, int64_t T);
// The cache rows of whole sequences one after the other: c [n][rank ld], key part [n][rot ld].
int32_t launch_latent_gather(kanso_cuda_ctx* ctx, const LatentAttn& a, const KvDenseLayer& kv,
                             const RowMap& map, const AttnTile* runs, uint32_t n_runs, bf16* c,
                             bf16* rot, int64_t n);
// Attention on the latents themselves. q_lat f32: row i's head h at i * q_row + h * q_head, rank
// columns (the query's unrotated part through the transposed key projection); out likewise,
// sum_j w_j c_j in f32 or the element type. rows: the row of the step that row i is (nullptr: i).
// early: every visible key but the rows' own was stored by earlier steps.
struct LatentRows {
  const float* q_lat = nullptr;
  int64_t q_row = 0, q_head = 0;
  LatentQuery q;  // for the rotated parts
  const uint32_t* rows = nullptr;
  RowMap map;
  uint32_t max_keys = 0;
  bool early = false;
  void* out = nullptr;
  bool out_f32 = false;
  int64_t out_row = 0, out_head = 0;
  int64_t n = 0;
};
// path 0: the library's choice, 1: plain, 2: mma tiles of 16 heads (bfloat16; *handled = false when a
// size is outside its range)
int32_t launch_latent_attn_rows(kanso_cuda_ctx* ctx, int32_t compute, const LatentAttn& a,
                                const KvDenseLayer& kv, const LatentRows& r, int path,
                                bool* handled);
// Causal softmax attention of prompts on tcgen05, bfloat16, over keys and values that lie one
// after the other: k [n][heads][dim ld] with rows of k_ld elements, v likewise, k_rot [n][rot ld]
// shared by the heads (rot 0: none); q and q_rot as launch_latent_q_rows leaves them. A tile's last
// word is where its sequence's keys begin. sink may be nullptr. *handled = false when a size is
// outside the kernel's range.
struct SoftmaxPrefill {
  uint32_t heads = 0, dim = 0, rot = 0, vdim = 0;
  float scale = 1.f;
  const float* sink = nullptr;
  const bf16 *q = nullptr, *q_rot = nullptr;
  int64_t q_rows = 0;
  const bf16 *k = nullptr, *v = nullptr, *k_rot = nullptr;
  int64_t k_ld = 0, v_ld = 0, keys = 0;
  const AttnTile* tiles = nullptr;
  uint32_t n_tiles = 0;
  bf16* out = nullptr;  // [rows][heads * vdim], rows of out_ld
  int64_t out_ld = 0;
};
bool softmax_prefill_fits(const SoftmaxPrefill& p);
int32_t launch_softmax_prefill(kanso_cuda_ctx* ctx, const SoftmaxPrefill& p, bool* handled);

// ---- matrix memory (csrc/mlstm.cu) ----
// The projections of a row, f32 as the sum of parts: [q | k | v | gate | i | f] with heads * dim,
// heads * dim, heads * vdim, heads * vdim, heads, heads columns.
struct MlstmArgs {
  uint32_t heads = 0, dim = 0, vdim = 0;
  float cap = 1.f;
  const float *i_bias = nullptr, *f_bias = nullptr;  // [heads]
  const float* y = nullptr;
  int parts = 1;
  int64_t part_stride = 0;
  KvStateLayer state;
  const uint32_t* positions = nullptr;
  const AttnTile* portions = nullptr;  // nullptr: row t is all of sequence t
  const uint32_t* slots = nullptr;     // per sequence; nullptr: s
  float* out = nullptr;                // [T][heads * vdim], not yet normed
  __host__ __device__ int64_t width() const {
    return (int64_t)heads * (2 * dim + 2 * vdim + 2);
  }
};
// n portions, token by token from the state that earlier steps left. max_rows bounds their length.
int32_t launch_mlstm_rows(kanso_cuda_ctx* ctx, const MlstmArgs& a, uint32_t n, uint32_t max_rows);
// n portions of at most max_rows tokens in chunks of 64 on the tensor cores; q, k, v are the bfloat16
// operands. mem: mlstm_chunk_bytes of workspace for T, the rows of the step.
bool mlstm_chunk_fits(const MlstmArgs& a);
size_t mlstm_chunk_bytes(uint32_t heads, uint32_t dim, uint32_t vdim, int64_t T);
int32_t launch_mlstm_chunks(kanso_cuda_ctx* ctx, const MlstmArgs& a, uint32_t n, uint32_t max_rows,
                            void* mem, int64_t T);
// out[t] = each head of o over its own root mean square, times w, times sigmoid(gate), in the
// products' element type; the gate lies in the projections' rows.
int32_t launch_head_norm_gate(kanso_cuda_ctx* ctx, int32_t compute, const MlstmArgs& a,
                              const float* w, float eps, void* out, int64_t out_ld, int64_t T);

}  // namespace kanso
