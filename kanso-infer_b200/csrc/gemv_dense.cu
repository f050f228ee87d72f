// Row-streaming products of unquantised weights (bfloat16 or f32) with one or two activation
// rows: the decode step of the models with bfloat16 weights.
//
// A warp (or KS warps that share the columns) takes four weight rows at a time; a lane reads 16
// bytes of each with the streaming path, the next 16 bytes requested before the current ones are
// used, and multiplies them with the activations in shared memory (f32). The activations' eight
// floats per lane step lie in two planes of four, so that the lanes' 16-byte reads are
// consecutive. Accumulators are reduced by a transposing butterfly: log2(32) exchanges of half the
// values each instead of five exchanges per value.
//
// Three kernels use that core: the plain product (with the residual step in front of it where the
// caller asks, so that a layer needs no norm launch), the experts' gate and up product with the
// routing decision in front of it, and the experts' down product, whose columns are the chosen
// experts' one after the other. A matrix of several groups (one per head) takes an input of its own
// for each.
#include <cmath>
#include <type_traits>

#include "dense.cuh"

namespace kanso {

constexpr int GV_THREADS = 256;
constexpr int GV_WARPS = GV_THREADS / 32;
constexpr int GV_ROWS = 4;  // weight rows per warp step

template <typename E>
using RawOf = decltype(load_raw(static_cast<const E*>(nullptr)));

__device__ __forceinline__ int xs_index(int i, int ld) {
  return ((i >> 2) & 1) * (ld >> 1) + (i >> 3) * 4 + (i & 3);
}

// acc[r * TT + t] += row r . x t over the chunks c0, c0 + step, ... (a chunk is 8 columns)
template <typename E, int TT>
__device__ __forceinline__ void dot_rows(const E* const (&row)[GV_ROWS], RawOf<E> (&cur)[GV_ROWS],
                                         int c0, int step, int chunks, const float* xs, int ld,
                                         float (&acc)[GV_ROWS * TT]) {
  for (int c = c0; c < chunks; c += step) {
    RawOf<E> next[GV_ROWS];
    const bool more = c + step < chunks;
    if (more) {
#pragma unroll
      for (int r = 0; r < GV_ROWS; ++r) next[r] = load_raw_once(row[r] + (size_t)(c + step) * 8);
    }
    float wv[GV_ROWS][8];
#pragma unroll
    for (int r = 0; r < GV_ROWS; ++r) expand(cur[r], wv[r]);
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      const float4 lo = *reinterpret_cast<const float4*>(xs + t * ld + c * 4);
      const float4 hi = *reinterpret_cast<const float4*>(xs + t * ld + (ld >> 1) + c * 4);
#pragma unroll
      for (int r = 0; r < GV_ROWS; ++r) {
        float s = acc[r * TT + t];
        s = fmaf(wv[r][0], lo.x, s);
        s = fmaf(wv[r][1], lo.y, s);
        s = fmaf(wv[r][2], lo.z, s);
        s = fmaf(wv[r][3], lo.w, s);
        s = fmaf(wv[r][4], hi.x, s);
        s = fmaf(wv[r][5], hi.y, s);
        s = fmaf(wv[r][6], hi.z, s);
        acc[r * TT + t] = fmaf(wv[r][7], hi.w, s);
      }
    }
    if (more) {
#pragma unroll
      for (int r = 0; r < GV_ROWS; ++r) cur[r] = next[r];
    }
  }
}

// Sums V values over the warp; lane l returns the sum of value l / (32 / V).
template <int V>
__device__ __forceinline__ float warp_sum_scatter(float (&v)[V], int lane) {
  int n = V;
#pragma unroll
  for (int o = 16; o; o >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = lane & o;
#pragma unroll
      for (int i = 0; i < V / 2; ++i) {
        if (i < n) {
          const float send = up ? v[i] : v[i + n];
          const float keep = up ? v[i + n] : v[i];
          v[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, o);
        }
      }
    } else {
      v[0] += __shfl_xor_sync(0xFFFFFFFFu, v[0], o);
    }
  }
  return v[0];
}

// Adds the KS warps' shares of a row group and hands each sum to `store(group, value index, sum)`.
// Every thread of the CTA must come here.
template <int V, typename F>
__device__ __forceinline__ void finish_rows(float (&acc)[V], int ks, float* red, F store) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float s = warp_sum_scatter<V>(acc, lane);
  constexpr int REP = 32 / V;
  if (ks == 1) {
    if (lane % REP == 0) store(warp, lane / REP, s);
    return;
  }
  if (lane % REP == 0) red[warp * V + lane / REP] = s;
  __syncthreads();
  for (int i = threadIdx.x; i < GV_WARPS / ks * V; i += GV_THREADS) {
    const int group = i / V, idx = i % V;
    float sum = 0.f;
    for (int k = 0; k < ks; ++k) sum += red[(group * ks + k) * V + idx];
    store(group, idx, sum);
  }
  __syncthreads();
}

// What a launch of the plain product's kernel is made for: rows with a residual step that adds and
// results as they are; rows with any residual step and results through GemvOut; inputs that lie in
// groups (and the store beside them); gated heads.
enum GemvKind { GV_PLAIN, GV_ROWS_IN, GV_GROUPS_IN, GV_GATED_IN };

struct GemvArgs {
  const void* w;
  int rows, cols, ld, ks, T;
  GemvSource s;
  float* out;
  int64_t out_ld;
  GemvOut o;
};
struct GemvStoreArgs : GemvArgs {
  int store_ctas;  // CTAs in front of the product's that store the step's cache rows
  LatentStore store;
};
template <int KIND>
using GemvArgsOf = std::conditional_t<KIND == GV_GROUPS_IN, GemvStoreArgs, GemvArgs>;

// Each head over its own root mean square, weight and gate (GemvSource::gate): a warp per head, or
// several where the heads are few. Every thread of the CTA must come here.
__device__ __forceinline__ void gate_source(const GemvSource& s, const float* x, const float* gate,
                                            int cols, int ld, float* xt, float* red) {
  const int hd = cols / s.heads, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int wph = 1;  // warps per head
  while (wph * 2 * s.heads <= GV_WARPS) wph *= 2;
  const int sub = warp % wph, step = wph * 32;
  for (int h0 = 0; h0 < s.heads; h0 += GV_WARPS / wph) {
    const int h = h0 + warp / wph;
    const int first = h * hd + sub * 32 + lane, end = h < s.heads ? (h + 1) * hd : 0;
    float ss = 0.f;
#pragma unroll 4
    for (int i = first; i < end; i += step) {
      const float v = x[i];
      float g = gate[i];
      for (int p = 1; p < s.parts; ++p) g += gate[p * s.part_stride + i];
      xt[xs_index(i, ld)] = v * s.norm_w[i] / (1.0f + expf(-g));
      ss += v * v;
    }
#pragma unroll
    for (int o = 16; o; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
    if (wph > 1) {
      if (lane == 0) red[warp] = ss;
      __syncthreads();
      ss = 0.f;
      for (int k = 0; k < wph; ++k) ss += red[warp - sub + k];
      __syncthreads();
    }
    const float inv = 1.0f / sqrtf(ss / (float)hd + s.eps);
#pragma unroll 4
    for (int i = first; i < end; i += step) xt[xs_index(i, ld)] *= inv;
  }
}

// The input rows of this CTA, into shared memory (and the residual step's to x_out by one CTA).
template <int TT, int KIND>
__device__ __forceinline__ void norm_source(const GemvSource& s, int cols, int ld, int t0, int nt,
                                            bool writer, float* xs, float* red) {
  for (int t = 0; t < nt; ++t) {
    const int64_t r = s.row_index ? s.row_index[t0 + t] : t0 + t;
    const float* x = s.x + r * cols;
    float* xt = xs + t * ld;
    if (KIND == GV_GATED_IN) {
      gate_source(s, x, s.gate + r * s.gate_ld, cols, ld, xt, red);
    } else {
      if (KIND == GV_GROUPS_IN) x = s.x + r * s.x_ld + blockIdx.z * s.x_group;
      const bool step = KIND != GV_GROUPS_IN && s.y;
      const bool after = KIND == GV_ROWS_IN && step && s.form == Residual::kAddNorm;
      float inv = 0.f;
      if (step) {
        const float* y = s.y + r * cols;
        float ss = 0.f;
        for (int i = threadIdx.x; i < cols; i += GV_THREADS) {
          float v = y[i];
          for (int p = 1; p < s.parts; ++p) v += y[p * s.part_stride + i];
          if (after) v = fmaf(s.mult, x[i], v);
          xt[xs_index(i, ld)] = v;
          ss += v * v;
        }
        ss = block_sum(ss, red);
        inv = 1.0f / sqrtf(ss / (float)cols + s.eps);
      }
      float s2 = 0.f;
      for (int i = threadIdx.x; i < cols; i += GV_THREADS) {
        float v = after ? 0.f : x[i];
        if (step) {
          const float n = xt[xs_index(i, ld)] * inv * s.norm_w[i];
          v = after ? n : v + s.mult * n;
        }
        xt[xs_index(i, ld)] = v;
        if (writer && s.x_out) s.x_out[r * cols + i] = v;
        s2 += v * v;
      }
      if (s.final_w) {
        s2 = block_sum(s2, red);
        const float inv2 = 1.0f / sqrtf(s2 / (float)cols + s.eps);
        for (int i = threadIdx.x; i < cols; i += GV_THREADS)
          xt[xs_index(i, ld)] = xt[xs_index(i, ld)] * inv2 * s.final_w[i];
      }
    }
    for (int i = cols + threadIdx.x; i < ld; i += GV_THREADS) xt[xs_index(i, ld)] = 0.f;
  }
  for (int t = nt; t < TT; ++t)
    for (int i = threadIdx.x; i < ld; i += GV_THREADS) xs[t * ld + i] = 0.f;
}

template <typename E, int TT, int KIND>
__global__ void __launch_bounds__(GV_THREADS, sizeof(E) == 2 ? (TT == 1 ? 4 : 3) : 2)
    gemv_dense_kernel(const GemvArgsOf<KIND> a) {
  extern __shared__ __align__(16) float xs[];
  __shared__ float red[GV_WARPS * GV_ROWS * TT > 32 ? GV_WARPS * GV_ROWS * TT : 32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gpc = GV_WARPS / a.ks, sub = warp % a.ks, chunks = a.ld / 8;
  const int t0 = blockIdx.y * TT, nt = min(TT, a.T - t0);
  const int groups = (a.rows + GV_ROWS - 1) / GV_ROWS;
  const E* w = static_cast<const E*>(a.w);
  float* out = a.out;
  int cta = blockIdx.x, ctas = gridDim.x;
  if constexpr (KIND == GV_GROUPS_IN) {
    if (cta < a.store_ctas) {
      pdl_launch_dependents();
      const float2 turn = latent_turn(a.store, cta);
      pdl_wait();
      if (blockIdx.y == 0 && blockIdx.z == 0) latent_store_row<E>(a.store, cta, turn, red);
      return;
    }
    cta -= a.store_ctas;
    ctas -= a.store_ctas;
    w += (int64_t)blockIdx.z * a.rows * a.ld;
    out += blockIdx.z * a.o.group_step;
  }
  const int c0 = sub * 32 + lane, step = a.ks * 32;
  const E* row[GV_ROWS];
  RawOf<E> cur[GV_ROWS];
  auto open_group = [&](int g) {
#pragma unroll
    for (int r = 0; r < GV_ROWS; ++r) {
      row[r] = w + (int64_t)min(min(g, groups - 1) * GV_ROWS + r, a.rows - 1) * a.ld;
      if (c0 < chunks) cur[r] = load_raw_once(row[r] + (size_t)c0 * 8);
    }
  };
  int base = cta * gpc;
  open_group(base + warp / a.ks);  // weights depend on nothing that runs before this kernel
  pdl_launch_dependents();
  pdl_wait();
  norm_source<TT, KIND>(a.s, a.cols, a.ld, t0, nt, cta == 0, xs, red);
  __syncthreads();
  while (true) {
    float acc[GV_ROWS * TT];
#pragma unroll
    for (int i = 0; i < GV_ROWS * TT; ++i) acc[i] = 0.f;
    dot_rows<E, TT>(row, cur, c0, step, chunks, xs, a.ld, acc);
    const int nbase = base + ctas * gpc;
    if (nbase < groups) open_group(nbase + warp / a.ks);
    finish_rows<GV_ROWS * TT>(acc, a.ks, red, [&](int grp, int idx, float v) {
      const int n = (base + grp) * GV_ROWS + idx / TT, t = idx % TT;
      if (n >= a.rows || t >= nt) return;
      if (KIND == GV_ROWS_IN) {
        if (a.o.bias) v += a.o.bias[n];
        if (a.o.relu2) v = relu_squared(v);
      }
      out[(int64_t)(t0 + t) * a.out_ld + n] = v;
    });
    if (nbase >= groups) break;
    base = nbase;
  }
}

struct GateUpArgs {
  const void *gate, *up;
  int ff, cols, ld, ff_ld, ks, top, experts;
  RouteWeights form;
  const float* x;
  const float* logits;
  float* act;
  uint32_t* sel;
};

// Two gate rows and the two up rows beside them per warp step, without a gate four up rows;
// blockIdx.y = row * top + place.
template <typename E, bool GATED>
__global__ void __launch_bounds__(GV_THREADS) gemv_gate_up_kernel(const GateUpArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[GV_WARPS * GV_ROWS];
  float* xs = sm;                          // [ld]
  float* lg = xs + a.ld;                   // [experts]
  float* wt = lg + a.experts;              // [top]
  uint32_t* sel = reinterpret_cast<uint32_t*>(wt + a.top);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.y / a.top, place = blockIdx.y % a.top;
  pdl_launch_dependents();
  pdl_wait();
  for (int e = threadIdx.x; e < a.experts; e += GV_THREADS)
    lg[e] = a.logits[(int64_t)t * a.experts + e];
  for (int i = threadIdx.x; i < a.ld; i += GV_THREADS)
    xs[xs_index(i, a.ld)] = i < a.cols ? a.x[(int64_t)t * a.cols + i] : 0.f;
  __syncthreads();
  if (warp == 0) warp_route(lg, a.experts, a.top, a.form, lane, sel, wt);
  __syncthreads();
  if (blockIdx.x == 0 && threadIdx.x == 0) a.sel[blockIdx.y] = sel[place];
  const float weight = wt[place];
  const int64_t ebase = (int64_t)sel[place] * a.ff;
  const int gpc = GV_WARPS / a.ks, sub = warp % a.ks, chunks = a.ld / 8;
  constexpr int PER = GATED ? 2 : 4;  // results per warp step
  const int c0 = sub * 32 + lane, groups = (a.ff + PER - 1) / PER;
  for (int base = blockIdx.x * gpc; base < groups; base += gridDim.x * gpc) {
    const int f0 = min(base + warp / a.ks, groups - 1) * PER;
    const E* row[GV_ROWS];
    RawOf<E> cur[GV_ROWS];
#pragma unroll
    for (int r = 0; r < GV_ROWS; ++r) {
      const E* m = static_cast<const E*>(GATED && r < 2 ? a.gate : a.up);
      row[r] = m + (ebase + min(f0 + (GATED ? r & 1 : r), a.ff - 1)) * a.ld;
      if (c0 < chunks) cur[r] = load_raw_once(row[r] + (size_t)c0 * 8);
    }
    float acc[GV_ROWS] = {0.f, 0.f, 0.f, 0.f};
    dot_rows<E, 1>(row, cur, c0, a.ks * 32, chunks, xs, a.ld, acc);
    const float s = warp_sum_scatter<GV_ROWS>(acc, lane);  // lane / 8 = row of the four
    if (lane % 8 == 0) red[warp * GV_ROWS + lane / 8] = s;
    __syncthreads();
    if (threadIdx.x < gpc * PER) {
      const int grp = threadIdx.x / PER, f = threadIdx.x % PER;
      float g = 0.f, u = 0.f;
      for (int k = 0; k < a.ks; ++k) {
        g += red[(grp * a.ks + k) * GV_ROWS + f];
        if (GATED) u += red[(grp * a.ks + k) * GV_ROWS + 2 + f];
      }
      const int n = (base + grp) * PER + f;
      if (base + grp < groups && n < a.ff)
        a.act[(int64_t)blockIdx.y * a.ff_ld + n] = weight * (GATED ? silu(g) * u : relu_squared(g));
    }
    __syncthreads();
  }
  if (blockIdx.x == 0)
    for (int n = a.ff + threadIdx.x; n < a.ff_ld; n += GV_THREADS)
      a.act[(int64_t)blockIdx.y * a.ff_ld + n] = 0.f;
}

struct DownArgs {
  const void* w;
  int rows, ld, ks, top;
  const float* act;
  const uint32_t* sel;
  float* out;
};

// blockIdx.y = row of the step; the columns are the chosen experts' one after the other.
template <typename E>
__global__ void __launch_bounds__(GV_THREADS) gemv_down_kernel(const DownArgs a) {
  extern __shared__ __align__(16) float xs[];  // [top][ld], two planes each
  __shared__ float red[GV_WARPS * GV_ROWS];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  for (int i = threadIdx.x; i < a.top * a.ld; i += GV_THREADS) {
    const int j = i / a.ld, c = i - j * a.ld;
    xs[j * a.ld + xs_index(c, a.ld)] = a.act[(int64_t)t * a.top * a.ld + i];
  }
  __syncthreads();
  const int gpc = GV_WARPS / a.ks, sub = warp % a.ks, per = a.ld / 8, chunks = per * a.top;
  const int groups = (a.rows + GV_ROWS - 1) / GV_ROWS;
  const uint32_t* sel = a.sel + (int64_t)t * a.top;
  for (int base = blockIdx.x * gpc; base < groups; base += gridDim.x * gpc) {
    const int g = min(base + warp / a.ks, groups - 1);
    int64_t roff[GV_ROWS];
#pragma unroll
    for (int r = 0; r < GV_ROWS; ++r)
      roff[r] = (int64_t)min(g * GV_ROWS + r, a.rows - 1) * a.ld;
    float acc[GV_ROWS] = {0.f, 0.f, 0.f, 0.f};
    const int step = a.ks * 32;
    auto fetch = [&](int cc, RawOf<E> (&raw)[GV_ROWS]) {
      const int j = cc / per, c = cc - j * per;
      const E* b = static_cast<const E*>(a.w) + (int64_t)sel[j] * a.rows * a.ld + (size_t)c * 8;
#pragma unroll
      for (int r = 0; r < GV_ROWS; ++r) raw[r] = load_raw_once(b + roff[r]);
    };
    RawOf<E> cur[GV_ROWS], next[GV_ROWS];
    int cc = sub * 32 + lane;
    if (cc < chunks) fetch(cc, cur);
    for (; cc < chunks; cc += step) {
      if (cc + step < chunks) fetch(cc + step, next);
      const int j = cc / per, c = cc - j * per;
      const float4 lo = *reinterpret_cast<const float4*>(xs + j * a.ld + c * 4);
      const float4 hi = *reinterpret_cast<const float4*>(xs + j * a.ld + (a.ld >> 1) + c * 4);
#pragma unroll
      for (int r = 0; r < GV_ROWS; ++r) {
        float wv[8];
        expand(cur[r], wv);
        float s = acc[r];
        s = fmaf(wv[0], lo.x, s);
        s = fmaf(wv[1], lo.y, s);
        s = fmaf(wv[2], lo.z, s);
        s = fmaf(wv[3], lo.w, s);
        s = fmaf(wv[4], hi.x, s);
        s = fmaf(wv[5], hi.y, s);
        s = fmaf(wv[6], hi.z, s);
        acc[r] = fmaf(wv[7], hi.w, s);
      }
#pragma unroll
      for (int r = 0; r < GV_ROWS; ++r) cur[r] = next[r];
    }
    finish_rows<GV_ROWS>(acc, a.ks, red, [&](int grp, int idx, float v) {
      const int n = (base + grp) * GV_ROWS + idx;
      if (base + grp < groups && n < a.rows) a.out[(int64_t)t * a.rows + n] = v;
    });
  }
}

// Warps that share a row group: enough CTAs for two per SM as long as every warp keeps at least
// two trips along the columns.
static int pick_ks(const kanso_cuda_ctx* ctx, int64_t groups, int64_t copies, int64_t chunks) {
  int ks = 1;
  while (ks < GV_WARPS && groups * ks * copies < (int64_t)2 * ctx->sm_count * GV_WARPS &&
         chunks >= ks * 2 * 32)
    ks *= 2;
  return ks;
}
static unsigned gv_grid(const kanso_cuda_ctx* ctx, int64_t groups, int ks, int64_t copies) {
  const int64_t gpc = GV_WARPS / ks, need = (groups + gpc - 1) / gpc;
  const int64_t cap = std::max<int64_t>(1, 8 * (int64_t)ctx->sm_count / copies);
  return (unsigned)std::min(need, cap);
}

template <typename E, int TT, int KIND>
static int32_t gemv_launch(kanso_cuda_ctx* ctx, const GemvArgsOf<KIND>& a, dim3 grid, size_t smem) {
  int32_t st = allow_max_smem(ctx, (const void*)gemv_dense_kernel<E, TT, KIND>);
  if (st) return st;
  const cudaError_t e =
      launch_dependent(ctx, gemv_dense_kernel<E, TT, KIND>, grid, dim3(GV_THREADS), smem, a);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "gemv_dense launch");
  return after_launch(ctx, "gemv_dense");
}
template <typename E, int TT>
static int32_t gemv_launch(kanso_cuda_ctx* ctx, const GemvStoreArgs& a, dim3 grid, size_t smem) {
  if (a.s.gate) return gemv_launch<E, TT, GV_GATED_IN>(ctx, a, grid, smem);
  if (a.s.x_ld) return gemv_launch<E, TT, GV_GROUPS_IN>(ctx, a, grid, smem);
  if (a.o.bias || a.o.relu2 || (a.s.y && a.s.form != Residual::kAdd))
    return gemv_launch<E, TT, GV_ROWS_IN>(ctx, a, grid, smem);
  return gemv_launch<E, TT, GV_PLAIN>(ctx, a, grid, smem);
}

int32_t launch_gemv(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat& w, const GemvSource& s,
                    float* out, int64_t out_ld, int T, const GemvOut& o, const LatentStore* store) {
  int tt = 1;
  while (tt < T && tt < GEMV_MAX_T && (int64_t)tt * 2 * w.ld * 4 <= 128 * 1024) tt *= 2;
  const size_t smem = (size_t)tt * w.ld * 4;
  if (smem > (size_t)GEMV_MAX_COLS * 4)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "dense product: %lld columns", (long long)w.cols);
  const int64_t groups = (w.rows + GV_ROWS - 1) / GV_ROWS, copies = (T + tt - 1) / tt;
  const int64_t all = copies * w.groups;
  if (w.groups > 65535 || ((w.groups > 1 || store) && (!s.x_ld || s.y)) ||
      ((s.x_ld || s.gate) && (o.bias || o.relu2)))
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "dense product: %lld groups", (long long)w.groups);
  GemvStoreArgs a;
  static_cast<GemvArgs&>(a) = {w.w, (int)w.rows, (int)w.cols, (int)w.ld,
                               pick_ks(ctx, groups, all, w.ld / 8), T, s, out, out_ld, o};
  a.store_ctas = store ? T : 0;
  if (store) a.store = *store;
  const dim3 grid(gv_grid(ctx, groups, a.ks, all) + a.store_ctas, (unsigned)copies,
                  (unsigned)w.groups);
  if (compute == KANSO_COMPUTE_BF16) {
    switch (tt) {
      case 1: return gemv_launch<bf16, 1>(ctx, a, grid, smem);
      default: return gemv_launch<bf16, 2>(ctx, a, grid, smem);
    }
  }
  switch (tt) {
    case 1: return gemv_launch<float, 1>(ctx, a, grid, smem);
    default: return gemv_launch<float, 2>(ctx, a, grid, smem);
  }
}

int32_t launch_gemv_gate_up(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat* gate,
                            const DenseMat& up, const float* x, const float* router_logits,
                            uint32_t experts, uint32_t top, RouteWeights form, float* act,
                            uint32_t* sel, int T) {
  const int64_t per = gate ? 2 : 4, groups = (up.rows + per - 1) / per, copies = (int64_t)T * top;
  GateUpArgs a = {gate ? gate->w : nullptr, up.w, (int)up.rows, (int)up.cols, (int)up.ld,
                  (int)round_up8(up.rows), pick_ks(ctx, groups, copies, up.ld / 8), (int)top,
                  (int)experts, form, x, router_logits, act, sel};
  const dim3 grid(gv_grid(ctx, groups, a.ks, copies), (unsigned)copies);
  const size_t smem = ((size_t)up.ld + experts + 2 * top) * 4;
  if (smem > (size_t)GEMV_MAX_COLS * 4)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "expert product: %lld columns, %u experts",
                (long long)up.cols, experts);
  const bool b16 = compute == KANSO_COMPUTE_BF16;
  auto kern = gate ? (b16 ? gemv_gate_up_kernel<bf16, true> : gemv_gate_up_kernel<float, true>)
                   : (b16 ? gemv_gate_up_kernel<bf16, false> : gemv_gate_up_kernel<float, false>);
  int32_t st = allow_max_smem(ctx, (const void*)kern);
  if (st) return st;
  const cudaError_t e = launch_dependent(ctx, kern, grid, dim3(GV_THREADS), smem, a);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "gemv_gate_up launch");
  return after_launch(ctx, "gemv_gate_up");
}

int32_t launch_gemv_down(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat& down,
                         const float* act, const uint32_t* sel, uint32_t top, float* out, int T) {
  const int64_t groups = (down.rows + GV_ROWS - 1) / GV_ROWS;
  DownArgs a = {down.w, (int)down.rows, (int)down.ld,
                pick_ks(ctx, groups, T, down.ld / 8 * top), (int)top, act, sel, out};
  const dim3 grid(gv_grid(ctx, groups, a.ks, T), (unsigned)T);
  const size_t smem = (size_t)top * down.ld * 4;
  if (smem > (size_t)GEMV_MAX_COLS * 4)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "expert product: %u experts of %lld columns", top,
                (long long)down.cols);
  auto kern = compute == KANSO_COMPUTE_BF16 ? gemv_down_kernel<bf16> : gemv_down_kernel<float>;
  int32_t st = allow_max_smem(ctx, (const void*)kern);
  if (st) return st;
  const cudaError_t e = launch_dependent(ctx, kern, grid, dim3(GV_THREADS), smem, a);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "gemv_down launch");
  return after_launch(ctx, "gemv_down");
}

}  // namespace kanso
