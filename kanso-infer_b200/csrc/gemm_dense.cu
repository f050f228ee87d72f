// Tile products of unquantised weights with many activation rows: prompts, batched decoding and
// the routed experts (grouped rows).
//
// bfloat16: a CTA computes 128 weight rows x NT activation rows (two weight tiles of 128 when
// DUAL), both operands K-major in the 128-byte swizzle, brought by tensor-map copies into a ring
// of shared-memory stages of 64 columns; one thread issues the copies, one the tcgen05.mma
// (kind::f16, M = 128, N = NT), accumulators in TMEM. The weights take the M side, so that a few
// activation rows need no padding to 128, and an epilogue warp writes 32 consecutive results of
// one activation row. DUAL either doubles the weight rows of a CTA or, for the experts, holds the
// gate and the up accumulator of the same row in the same TMEM lane, so that silu(gate) * up is
// formed in the epilogue.
//
// Grouped rows: the activation rows are sorted by group (expert); the grid covers the most tiles
// there can be and a CTA finds its (group, tile) from the offsets on the device, so the host
// never waits for the routing. A tile that runs past its group's end computes rows of the next
// group and does not store them.
//
// f32: 64 x 64 tiles on the FMA units.
#include <algorithm>
#include <type_traits>

#include "dense.cuh"
#include "tc05.cuh"
#include "tensor_map.h"

namespace kanso {

constexpr int GD_THREADS = 128;
constexpr int GD_K = 64;  // columns per stage (128 bytes)
constexpr int GD_A_BYTES = 128 * 128;

struct GemmDenseArgs {
  void* out;            // f32 results, or the element type for the experts' activations
  int64_t out_ld, part_stride;
  const uint32_t* offsets;
  int64_t T;
  int groups, rows, k_steps, steps_per_split;
  int* status;
  const float* bias;
  int64_t group_step;
  const uint32_t* row_list;
  int relu2, elem, n_end;  // n_end: columns that are written

  // The bias of column n, added once where the columns' sum is split.
  __device__ __forceinline__ float bias_of(int n) const {
    return bias && n < rows && blockIdx.z == 0 ? bias[n] : 0.f;
  }
};
// Where the rows of a tile's group go: row r at r * out_ld + shift, by the list if there is one.
struct RowPlace {
  int64_t shift = 0, first = 0;
  const uint32_t* list = nullptr;
  __device__ __forceinline__ RowPlace(const GemmDenseArgs& a, int group) {
    if (!a.group_step) return;
    const int64_t per = (uint32_t)a.T / (uint32_t)a.groups;
    shift = group * (a.row_list ? a.group_step : a.group_step - per * a.out_ld);
    first = group * per;
    list = a.row_list;
  }
  __device__ __forceinline__ int64_t at(int64_t row, int64_t out_ld) const {
    return (list ? (int64_t)list[row - first] : row) * out_ld + shift;
  }
};

// The (group, first row, end of the group) of tile `tile`; one warp. false: past the last tile.
__device__ __forceinline__ bool find_tile(const uint32_t* offsets, int groups, int64_t T, int nt,
                                          int tile, int lane, int* group, int64_t* first,
                                          int64_t* end) {
  if (!offsets) {
    if (groups == 1) {
      *group = 0;
      *first = (int64_t)tile * nt;
      *end = T;
      return *first < T;
    }
    const uint32_t per = (uint32_t)T / (uint32_t)groups, tiles = (per + nt - 1) / (uint32_t)nt;
    const uint32_t g = (uint32_t)tile / tiles;
    *group = (int)g;
    *first = (int64_t)g * per + (int64_t)((uint32_t)tile - g * tiles) * nt;
    *end = (int64_t)(g + 1) * per;
    return g < (uint32_t)groups;
  }
  int before = 0;
  for (int g0 = 0; g0 < groups; g0 += 32) {
    const int g = g0 + lane;
    const uint32_t b = g < groups ? offsets[g] : 0u, e = g < groups ? offsets[g + 1] : 0u;
    const int n = (int)((e - b + nt - 1) / nt);
    int incl = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xFFFFFFFFu, incl, o);
      if (lane >= o) incl += v;
    }
    const unsigned hit = __ballot_sync(0xFFFFFFFFu, before + incl > tile);
    if (hit) {
      const int l = __ffs(hit) - 1;
      const int tiles_before = before + __shfl_sync(0xFFFFFFFFu, incl - n, l);
      const uint32_t gb = __shfl_sync(0xFFFFFFFFu, b, l), ge = __shfl_sync(0xFFFFFFFFu, e, l);
      *group = g0 + l;
      *first = (int64_t)gb + (int64_t)(tile - tiles_before) * nt;
      *end = ge;
      return true;
    }
    before += __shfl_sync(0xFFFFFFFFu, incl, 31);
  }
  return false;
}

template <int NT, bool DUAL, bool ACT>
struct GdShape {
  static constexpr int kStage = GD_A_BYTES * (DUAL ? 2 : 1) + NT * 128;
  // two CTAs per SM for the single form, one for the dual form
  static constexpr int kStages = DUAL ? (NT <= 32 ? 5 : 4) : NT <= 32 ? 5 : NT <= 64 ? 4 : 3;
  static constexpr int kCols = (DUAL ? 2 : 1) * NT;
  static constexpr size_t kSmem = (size_t)kStage * kStages + 1024;
};

// The results of column n (and n + 128) through bias and activation to their places.
template <int NT, bool DUAL, typename O>
__device__ __forceinline__ void ext_rows(const GemmDenseArgs& a, const RowPlace& place, O* out,
                                         uint32_t tmem, int n, int64_t first, int valid) {
  const float b0 = a.bias_of(n), b1 = DUAL ? a.bias_of(n + 128) : 0.f;
  const bool in0 = n < a.n_end, in1 = DUAL && n + 128 < a.n_end, sq = a.relu2;
  const float low = sq ? 0.f : -INFINITY;
  const int64_t ld = a.out_ld;
  out += place.shift + n;
  for (int c = 0; c < NT; c += 16) {
    if (c >= valid) break;
    uint32_t r0[16], r1[16];
    tmem_ld16(tmem + c, r0);
    if (DUAL) tmem_ld16(tmem + NT + c, r1);
    O* o = out + (first + c) * ld;
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      if (c + j >= valid) continue;
      const float x = fmaxf(__uint_as_float(r0[j]) + b0, low);
      O* at = place.list ? out + place.list[first + c + j - place.first] * ld : o + j * ld;
      if (in0) at[0] = to_elem<O>(sq ? x * x : x);
      if (DUAL) {
        const float y = fmaxf(__uint_as_float(r1[j]) + b1, low);
        if (in1) at[128] = to_elem<O>(sq ? y * y : y);
      }
    }
  }
}

// EXT: results go through bias, activation, element type or place (GemmOut).
template <int NT, bool DUAL, bool ACT, bool EXT>
__global__ void __launch_bounds__(GD_THREADS)
    gemm_dense_kernel(const __grid_constant__ CUtensorMap wmap,
                      const __grid_constant__ CUtensorMap wmap2,
                      const __grid_constant__ CUtensorMap xmap, const GemmDenseArgs a) {
  using S = GdShape<NT, DUAL, ACT>;
  extern __shared__ uint8_t raw[];
  __shared__ uint64_t full[S::kStages], empty[S::kStages], acc_full;
  __shared__ uint32_t tmem_slot;
  __shared__ int tile_ok, tile_group;
  __shared__ int64_t tile_first, tile_end;
  __shared__ volatile int abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  uint8_t* ring = raw + ((1024u - (smem_u32(raw) & 1023u)) & 1023u);

  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    for (int i = 0; i < S::kStages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(&acc_full, 1);
    mbar_fence_init();
    abort_flag = 0;
  }
  pdl_wait();
  if (warp == 0) {
    int g = 0;
    int64_t f = 0, e = 0;
    const bool ok = find_tile(a.offsets, a.groups, a.T, NT, blockIdx.y, lane, &g, &f, &e);
    if (lane == 0) {
      tile_ok = ok;
      tile_group = g;
      tile_first = f;
      tile_end = e;
    }
  }
  __syncthreads();
  if (!tile_ok) return;
  if (warp == 1) tmem_alloc(&tmem_slot, S::kCols < 32 ? 32 : S::kCols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  const int n0 = blockIdx.x * 128 * (DUAL && !ACT ? 2 : 1);
  const int k0 = blockIdx.z * a.steps_per_split;
  const int k1 = min(k0 + a.steps_per_split, a.k_steps);

  if (warp == 0) {
    if (lane == 0) {
      int issued = 0;
      for (int k = k0, i = 0; k < k1; ++k, ++i) {
        const int s = i % S::kStages;
        if (!mbar_wait_bounded(&empty[s], ((uint32_t)(i / S::kStages) & 1u) ^ 1u) || abort_flag) {
          abort_flag = 1;
          break;
        }
        uint8_t* st = ring + s * S::kStage;
        mbar_arrive_expect_tx(&full[s], S::kStage);
        tma_load_3d(st, &wmap, k * GD_K, n0, tile_group, &full[s]);
        if (DUAL)
          tma_load_3d(st + GD_A_BYTES, ACT ? &wmap2 : &wmap, k * GD_K, ACT ? n0 : n0 + 128,
                      tile_group, &full[s]);
        tma_load_2d(st + GD_A_BYTES * (DUAL ? 2 : 1), &xmap, k * GD_K, (int)tile_first, &full[s]);
        issued = i + 1;
      }
      // leave only when every copy this thread started has landed (bounded)
      for (int i = max(0, issued - S::kStages); i < issued; ++i)
        mbar_wait_bounded(&full[i % S::kStages], (uint32_t)(i / S::kStages) & 1u);
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_n = NT;
      const uint32_t idesc = tc_idesc_bf16(128, idesc_n);
      bool ok = true;
      for (int k = k0, i = 0; k < k1; ++k, ++i) {
        const int s = i % S::kStages;
        if (!mbar_wait_bounded(&full[s], (uint32_t)(i / S::kStages) & 1u)) {
          ok = false;
          break;
        }
        tc_fence_after();
        const uint32_t base = smem_u32(ring + s * S::kStage);
        const uint64_t ad = tc_smem_desc_sw128(base);
        const uint64_t ad2 = tc_smem_desc_sw128(base + GD_A_BYTES);
        const uint64_t bd = tc_smem_desc_sw128(base + GD_A_BYTES * (DUAL ? 2 : 1));
#pragma unroll
        for (int j = 0; j < GD_K / 16; ++j) {
          const uint32_t acc = (i > 0 || j > 0) ? 1u : 0u;
          tc_mma_f16(tmem, ad + 2 * j, bd + 2 * j, idesc, acc);
          if (DUAL) tc_mma_f16(tmem + NT, ad2 + 2 * j, bd + 2 * j, idesc, acc);
        }
        tc_commit(&empty[s]);
      }
      if (ok)
        tc_commit(&acc_full);
      else
        abort_flag = 1;
    }
    __syncwarp();
  }
  __syncthreads();
  int failed = abort_flag != 0;
  if (!failed) failed = !mbar_wait_bounded(&acc_full, 0);
  failed = __syncthreads_or(failed);
  tc_fence_after();
  if (!failed) {
    const int n = n0 + warp * 32 + lane;  // a warp reaches its own quarter of the TMEM lanes
    const uint32_t lane_base = tmem + ((uint32_t)(warp * 32) << 16);
    const int valid = (int)min((int64_t)NT, tile_end - tile_first);
    if (EXT) {
      const RowPlace place(a, tile_group);
      if (a.elem)
        ext_rows<NT, DUAL>(a, place, static_cast<bf16*>(a.out), lane_base, n, tile_first, valid);
      else
        ext_rows<NT, DUAL>(a, place, static_cast<float*>(a.out) + (int64_t)blockIdx.z * a.part_stride,
                           lane_base, n, tile_first, valid);
    }
    for (int c = 0; c < NT / 16 && !EXT; ++c) {
      if (c * 16 >= valid) break;
      uint32_t r0[16], r1[16];
      tmem_ld16(lane_base + c * 16, r0);
      if (DUAL) tmem_ld16(lane_base + NT + c * 16, r1);
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        const int m = c * 16 + j;
        if (m >= valid) continue;
        const int64_t row = tile_first + m;
        if (ACT) {
          // the pad columns multiply weight rows that were zero-filled: they come out as zero
          const float g = __uint_as_float(r0[j]), u = __uint_as_float(r1[j]);
          if (n < a.out_ld)
            static_cast<bf16*>(a.out)[row * a.out_ld + n] = to_elem<bf16>(silu(g) * u);
        } else {
          float* o = static_cast<float*>(a.out) + (int64_t)blockIdx.z * a.part_stride +
                     row * a.out_ld;
          if (n < a.rows) o[n] = __uint_as_float(r0[j]);
          if (DUAL && n + 128 < a.rows) o[n + 128] = __uint_as_float(r1[j]);
        }
      }
    }
  } else if (threadIdx.x == 0) {
    atomicOr(a.status, DEV_WAIT_TIMEOUT);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, S::kCols < 32 ? 32 : S::kCols);
}

// ---- f32 ----
constexpr int GF_TILE = 64, GF_K = 16;

template <bool ACT>
__global__ void __launch_bounds__(256)
    gemm_f32_kernel(const float* __restrict__ w, const float* __restrict__ w2,
                    const float* __restrict__ x, int ld, const GemmDenseArgs a) {
  __shared__ float ws[GF_K][GF_TILE + 4], us[ACT ? GF_K : 1][GF_TILE + 4],
      xs[GF_K][GF_TILE + 4];
  __shared__ int tile_ok, tile_group;
  __shared__ int64_t tile_first, tile_end;
  pdl_launch_dependents();
  pdl_wait();
  if (threadIdx.x < 32) {
    int g = 0;
    int64_t f = 0, e = 0;
    const bool ok = find_tile(a.offsets, a.groups, a.T, GF_TILE, blockIdx.y, threadIdx.x, &g, &f, &e);
    if (threadIdx.x == 0) {
      tile_ok = ok;
      tile_group = g;
      tile_first = f;
      tile_end = e;
    }
  }
  __syncthreads();
  if (!tile_ok) return;
  const int n0 = blockIdx.x * GF_TILE;
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;  // tx: weight rows, ty: activation rows
  const float* wg = w + (int64_t)tile_group * a.rows * ld;
  const float* ug = ACT ? w2 + (int64_t)tile_group * a.rows * ld : nullptr;
  float acc[4][4] = {}, acu[4][4] = {};
  const int lr = threadIdx.x / 4, lk = threadIdx.x % 4 * 4;  // one float4 per matrix and thread
  for (int k = 0; k < ld; k += GF_K) {
    float4 wv = {0.f, 0.f, 0.f, 0.f}, uv = wv, xv = wv;
    const bool in = k + lk < ld;
    if (in && n0 + lr < a.rows)
      wv = *reinterpret_cast<const float4*>(wg + (int64_t)(n0 + lr) * ld + k + lk);
    if (ACT && in && n0 + lr < a.rows)
      uv = *reinterpret_cast<const float4*>(ug + (int64_t)(n0 + lr) * ld + k + lk);
    if (in && tile_first + lr < tile_end)
      xv = *reinterpret_cast<const float4*>(x + (tile_first + lr) * ld + k + lk);
    __syncthreads();
    ws[lk][lr] = wv.x, ws[lk + 1][lr] = wv.y, ws[lk + 2][lr] = wv.z, ws[lk + 3][lr] = wv.w;
    xs[lk][lr] = xv.x, xs[lk + 1][lr] = xv.y, xs[lk + 2][lr] = xv.z, xs[lk + 3][lr] = xv.w;
    if (ACT) us[lk][lr] = uv.x, us[lk + 1][lr] = uv.y, us[lk + 2][lr] = uv.z, us[lk + 3][lr] = uv.w;
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < GF_K; ++kk) {
      float wr[4], ur[4], xr[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        wr[i] = ws[kk][tx + 16 * i];
        if (ACT) ur[i] = us[kk][tx + 16 * i];
        xr[i] = xs[kk][ty + 16 * i];
      }
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          acc[m][i] = fmaf(wr[i], xr[m], acc[m][i]);
          if (ACT) acu[m][i] = fmaf(ur[i], xr[m], acu[m][i]);
        }
    }
  }
  const RowPlace place(a, tile_group);
#pragma unroll
  for (int m = 0; m < 4; ++m) {
    const int64_t row = tile_first + ty + 16 * m;
    if (row >= tile_end) continue;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int n = n0 + tx + 16 * i;
      if (ACT) {
        if (n < a.out_ld)
          static_cast<float*>(a.out)[row * a.out_ld + n] = silu(acc[m][i]) * acu[m][i];
      } else if (n < a.n_end) {
        const float v = acc[m][i] + a.bias_of(n);
        static_cast<float*>(a.out)[place.at(row, a.out_ld) + n] = a.relu2 ? relu_squared(v) : v;
      }
    }
  }
}

// [groups][rows][ld] in boxes of 128 rows x 64 columns
static int32_t weight_map(kanso_cuda_ctx* ctx, const DenseMat& w, CUtensorMap* map) {
  TmEncodeFn encode = tm_encoder();
  if (!encode) return fail(ctx, KANSO_ERR_DEVICE, "the driver has no tensor-map encoder");
  const cuuint64_t dim[3] = {(cuuint64_t)w.cols, (cuuint64_t)w.rows, (cuuint64_t)w.groups};
  const cuuint64_t stride[2] = {(cuuint64_t)w.ld * 2, (cuuint64_t)(w.rows * w.ld) * 2};
  const cuuint32_t box[3] = {GD_K, 128, 1}, es[3] = {1, 1, 1};
  if (encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, w.w, dim, stride, box, es,
             CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
             CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return fail(ctx, KANSO_ERR_DEVICE, "tensor map of a [%lld x %lld] weight", (long long)w.rows,
                (long long)w.cols);
  return KANSO_OK;
}
// [T][ld] in boxes of nt rows x 64 columns
static int32_t rows_map(kanso_cuda_ctx* ctx, const void* x, int64_t T, int64_t cols, int64_t ld,
                        int nt, CUtensorMap* map) {
  TmEncodeFn encode = tm_encoder();
  if (!encode) return fail(ctx, KANSO_ERR_DEVICE, "the driver has no tensor-map encoder");
  const cuuint64_t dim[2] = {(cuuint64_t)cols, (cuuint64_t)T};
  const cuuint64_t stride[1] = {(cuuint64_t)ld * 2};
  const cuuint32_t box[2] = {GD_K, (cuuint32_t)nt}, es[2] = {1, 1};
  if (encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(x), dim, stride, box, es,
             CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
             CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return fail(ctx, KANSO_ERR_DEVICE, "tensor map of [%lld x %lld] activations", (long long)T,
                (long long)cols);
  return KANSO_OK;
}

template <int NT, bool DUAL, bool ACT, bool EXT>
static int32_t gd_launch(kanso_cuda_ctx* ctx, dim3 grid, const CUtensorMap& wm,
                         const CUtensorMap& wm2, const CUtensorMap& xm, const GemmDenseArgs& a) {
  auto kern = gemm_dense_kernel<NT, DUAL, ACT, EXT>;
  int32_t st = allow_max_smem(ctx, (const void*)kern);
  if (st) return st;
  const cudaError_t e = launch_dependent(ctx, kern, grid, dim3(GD_THREADS),
                                         GdShape<NT, DUAL, ACT>::kSmem, wm, wm2, xm, a);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "gemm_dense launch");
  return after_launch(ctx, "gemm_dense");
}

// Tiles that cover the rows: exact for one group, the most there can be for several.
static int64_t tiles_of(const GemmRows& r, int nt) {
  if (!r.offsets) return r.groups * ((r.T / r.groups + nt - 1) / nt);
  return std::min<int64_t>((r.T + nt - 1) / nt + r.groups - 1, r.T);
}
static int pick_nt(const GemmRows& r) {
  const int64_t per = (r.T + r.groups - 1) / r.groups;
  const int64_t aim = r.offsets ? per + per / 2 : per;
  return aim <= 16 ? 16 : aim <= 32 ? 32 : aim <= 64 ? 64 : 128;
}

int32_t launch_gemm(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat& w, const void* x, void* y,
                    int64_t y_ld, const GemmRows& r, int max_splits, int* splits,
                    int64_t part_stride, const GemmOut& o) {
  *splits = 1;
  if (o.relu2 || o.elem) max_splits = 1;
  // pad columns of a result in element type belong to it unless the next group lies behind it
  const int n_end = (int)(o.elem && !o.group_step ? std::max<int64_t>(y_ld, w.rows) : w.rows);
  GemmDenseArgs a = {y, y_ld, part_stride, r.offsets, r.T, r.groups, (int)w.rows, 0, 0,
                     ctx->dev_status, o.bias, o.group_step, o.rows, o.relu2, o.elem, n_end};
  if (compute == KANSO_COMPUTE_F32) {
    const dim3 grid((unsigned)((w.rows + GF_TILE - 1) / GF_TILE), (unsigned)tiles_of(r, GF_TILE));
    const cudaError_t e =
        launch_dependent(ctx, gemm_f32_kernel<false>, grid, dim3(256), 0, (const float*)w.w,
                         (const float*)nullptr, (const float*)x, (int)w.ld, a);
    if (e != cudaSuccess) return cuda_fail(ctx, e, "gemm_f32 launch");
    return after_launch(ctx, "gemm_f32");
  }
  const int nt = pick_nt(r);
  CUtensorMap wm, xm;
  int32_t st = weight_map(ctx, w, &wm);
  if (!st) st = rows_map(ctx, x, r.T, w.cols, w.ld, nt, &xm);
  if (st) return st;
  const int64_t ty = tiles_of(r, nt), tx = (w.rows + 127) / 128;
  a.k_steps = (int)((w.cols + GD_K - 1) / GD_K);
  // short products spend more time on their ends than the second tile saves: there two CTAs per
  // SM, of which one stores while the other multiplies
  const bool dual = nt == 128 && tx * ty >= 4 * (int64_t)ctx->sm_count && a.k_steps >= 12;
  // a share of the columns per CTA while the grid stays within one wave of two CTAs per SM
  int sp = 1;
  while (sp * 2 <= max_splits && tx * ty * sp * 2 <= 2 * (int64_t)ctx->sm_count &&
         a.k_steps / (sp * 2) >= 4)
    sp *= 2;
  a.steps_per_split = (a.k_steps + sp - 1) / sp;
  sp = (a.k_steps + a.steps_per_split - 1) / a.steps_per_split;
  *splits = sp;
  const bool ext = o.bias || o.relu2 || o.elem || o.group_step;
  auto launch = [&](auto n, auto two, dim3 grid) {
    constexpr int NT = decltype(n)::value;
    constexpr bool DUAL = decltype(two)::value;
    return ext ? gd_launch<NT, DUAL, false, true>(ctx, grid, wm, wm, xm, a)
               : gd_launch<NT, DUAL, false, false>(ctx, grid, wm, wm, xm, a);
  };
  using std::integral_constant;
  if (dual)
    return launch(integral_constant<int, 128>(), std::true_type(),
                  dim3((unsigned)((w.rows + 255) / 256), (unsigned)ty, (unsigned)sp));
  const dim3 grid((unsigned)tx, (unsigned)ty, (unsigned)sp);
  switch (nt) {
    case 16: return launch(integral_constant<int, 16>(), std::false_type(), grid);
    case 32: return launch(integral_constant<int, 32>(), std::false_type(), grid);
    case 64: return launch(integral_constant<int, 64>(), std::false_type(), grid);
    default: return launch(integral_constant<int, 128>(), std::false_type(), grid);
  }
}

int32_t launch_gemm_gate_up(kanso_cuda_ctx* ctx, int32_t compute, const DenseMat& gate,
                            const DenseMat& up, const void* x, void* act, int64_t act_ld,
                            const GemmRows& r) {
  GemmDenseArgs a = {act, act_ld, 0, r.offsets, r.T, r.groups, (int)gate.rows, 0, 0,
                     ctx->dev_status, nullptr, 0, nullptr, 0, 0, 0};
  if (compute == KANSO_COMPUTE_F32) {
    const dim3 grid((unsigned)((gate.rows + GF_TILE - 1) / GF_TILE),
                    (unsigned)tiles_of(r, GF_TILE));
    const cudaError_t e =
        launch_dependent(ctx, gemm_f32_kernel<true>, grid, dim3(256), 0, (const float*)gate.w,
                         (const float*)up.w, (const float*)x, (int)gate.ld, a);
    if (e != cudaSuccess) return cuda_fail(ctx, e, "gemm_f32 launch");
    return after_launch(ctx, "gemm_f32");
  }
  const int nt = pick_nt(r);
  CUtensorMap gm, um, xm;
  int32_t st = weight_map(ctx, gate, &gm);
  if (!st) st = weight_map(ctx, up, &um);
  if (!st) st = rows_map(ctx, x, r.T, gate.cols, gate.ld, nt, &xm);
  if (st) return st;
  a.k_steps = a.steps_per_split = (int)((gate.cols + GD_K - 1) / GD_K);
  const dim3 grid((unsigned)((gate.rows + 127) / 128), (unsigned)tiles_of(r, nt));
  switch (nt) {
    case 16: return gd_launch<16, true, true, false>(ctx, grid, gm, um, xm, a);
    case 32: return gd_launch<32, true, true, false>(ctx, grid, gm, um, xm, a);
    case 64: return gd_launch<64, true, true, false>(ctx, grid, gm, um, xm, a);
    default: return gd_launch<128, true, true, false>(ctx, grid, gm, um, xm, a);
  }
}

}  // namespace kanso
