// Softmax attention on cached latents, for decoding and short portions. A token's cache row is
// [c | k_rot]; with the query's unrotated part taken through the transposed key projection
// beforehand (q_lat = W_uk^T q) and the value projection applied afterwards, every head reads the
// same rows:
//
//   s = scale * (q_lat . c_j + q_rot . k_rot_j),  0 <= j <= i
//   out = sum_j exp(s_j) c_j / (sum_j exp(s_j) + exp(sink))
//
// latent_rows: four heads per CTA, any size, f32 and (sizes beyond the other) bfloat16.
// latent_group: bfloat16, sixteen heads as the rows of an mma tile, 32 keys at a time; a staged row
// serves as key and as value. A row's keys may be shared out over several CTAs, which leave partial
// sums with their maxima; latent_merge adds them in order.
#include <algorithm>
#include <cmath>

#include "dense.cuh"
#include "tc05.cuh"
#include "tensor_map.h"
#include "warp_mma.cuh"

namespace kanso {

struct LatentRowsArgs {
  LatentAttn a;
  KvDenseLayer kv;
  LatentRows r;
  float* partial;  // parts > 1: [n][heads][parts][rec]: sums, maximum, denominator
  uint32_t parts, tile, rec;
  int stages;
  int* status;
};

// What a row's CTA knows before it waits for the kernel in front.
struct LatentSpan {
  int64_t t;
  uint32_t pos, k_begin, k_end, n_parts;
  const uint32_t* table;
};
__device__ __forceinline__ LatentSpan latent_span(const LatentRowsArgs& p, int64_t i,
                                                  uint32_t part) {
  LatentSpan s;
  s.t = p.r.rows ? p.r.rows[i] : i;
  s.pos = p.r.map.positions[s.t];
  const uint32_t seq = p.r.map.row_seq ? p.r.map.row_seq[s.t] : (uint32_t)s.t;
  s.table = p.r.map.tables + (size_t)seq * p.r.map.max_blocks;
  const uint32_t n_tiles = (s.pos + p.tile) / p.tile;       // tiles that hold keys 0 .. pos
  const uint32_t per = (n_tiles + p.parts - 1) / p.parts;   // tiles per share
  s.n_parts = (n_tiles + per - 1) / per;                    // shares that have keys
  s.k_begin = part * per * p.tile;
  s.k_end = min(s.pos + 1, s.k_begin + per * p.tile);
  return s;
}
__device__ __forceinline__ float latent_q_value(const LatentQuery& q, int64_t at) {
  float v = q.q[at];
  for (int p = 1; p < q.parts; ++p) v += q.q[p * q.part_stride + at];
  return v;
}
template <typename E>
__device__ __forceinline__ void latent_out(const LatentRowsArgs& p, int64_t i, int h, int c,
                                           float v) {
  const int64_t at = i * p.r.out_row + h * p.r.out_head + c;
  if (p.r.out_f32)
    static_cast<float*>(p.r.out)[at] = v;
  else
    static_cast<E*>(p.r.out)[at] = to_elem<E>(v);
}

// The shares of one head of one row (blockIdx.x, blockIdx.y), 128 columns at a time (blockIdx.z and
// on): a thread takes four of them from every eighth share.
constexpr int LM_THREADS = 256, LM_COLS = 128, LM_GROUPS = LM_THREADS / (LM_COLS / 4);
template <typename E>
__global__ void __launch_bounds__(LM_THREADS) latent_merge_kernel(const LatentRowsArgs p) {
  extern __shared__ float weight[];  // [parts], then the shares' denominators
  __shared__ __align__(16) float4 sums[LM_GROUPS][LM_COLS / 4];
  pdl_launch_dependents();
  const int h = blockIdx.x, R = p.a.rank, tid = threadIdx.x;
  const int64_t i = blockIdx.y;
  const uint32_t n = latent_span(p, i, 0).n_parts;
  const float* src = p.partial + ((size_t)i * p.a.heads + h) * p.parts * p.rec;
  float* dens = weight + p.parts;
  const int q = tid % (LM_COLS / 4), g = tid / (LM_COLS / 4);
  pdl_wait();
  float4 o[4];
  auto first_shares = [&](int c) {
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const uint32_t at = g + k * LM_GROUPS;
      o[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (at < n && c < R) o[k] = *reinterpret_cast<const float4*>(src + (size_t)at * p.rec + c);
    }
  };
  first_shares(blockIdx.z * LM_COLS + q * 4);  // on their way while the weights are formed
  for (uint32_t k = tid; k < n; k += LM_THREADS) {
    const float2 m = *reinterpret_cast<const float2*>(src + (size_t)k * p.rec + p.rec - 4);
    weight[k] = m.x;
    dens[k] = m.y;
  }
  __syncthreads();
  if (tid < 32) {
    const float sink = p.a.sink[h];
    float top = sink, den = 0.f;
    for (uint32_t k = tid; k < n; k += 32) top = fmaxf(top, weight[k]);
#pragma unroll
    for (int s = 16; s; s >>= 1) top = fmaxf(top, __shfl_xor_sync(0xFFFFFFFFu, top, s));
    for (uint32_t k = tid; k < n; k += 32) {
      weight[k] = expf(weight[k] - top);
      den += weight[k] * dens[k];
    }
#pragma unroll
    for (int s = 16; s; s >>= 1) den += __shfl_xor_sync(0xFFFFFFFFu, den, s);
    const float inv = 1.0f / (den + expf(sink - top));
    for (uint32_t k = tid; k < n; k += 32) weight[k] *= inv;
  }
  __syncthreads();
  for (int c0 = blockIdx.z * LM_COLS; c0 < R; c0 += gridDim.z * LM_COLS) {
    const int c = c0 + q * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    for (uint32_t k0 = g; k0 < n; k0 += 4 * LM_GROUPS) {
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const uint32_t at = k0 + k * LM_GROUPS;
        if (at < n) {  // the pad behind the last column may hold anything
          const float w = weight[at];
          v.x = fmaf(w, o[k].x, v.x), v.y = fmaf(w, o[k].y, v.y);
          v.z = fmaf(w, o[k].z, v.z), v.w = fmaf(w, o[k].w, v.w);
        }
        const uint32_t next = at + 4 * LM_GROUPS;
        if (next < n && c < R)
          o[k] = *reinterpret_cast<const float4*>(src + (size_t)next * p.rec + c);
      }
    }
    first_shares(c + gridDim.z * LM_COLS);
    sums[g][q] = v;
    __syncthreads();
    const int col = c0 + tid;
    if (tid < LM_COLS && col < R) {
      float t = 0.f;
#pragma unroll
      for (int k = 0; k < LM_GROUPS; ++k) t += reinterpret_cast<const float*>(sums[k])[tid];
      latent_out<E>(p, i, h, col, t);
    }
    __syncthreads();
  }
}

// ------------------------------------------------------------------------ any size ----
constexpr int LR_THREADS = 128, LR_HEADS = 4, LR_TILE = 32;

template <typename E>
__global__ void __launch_bounds__(LR_THREADS) latent_rows_kernel(const LatentRowsArgs p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float prob[LR_HEADS][LR_TILE], corr[LR_HEADS];
  __shared__ size_t key_at[LR_TILE];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int part = blockIdx.x, h0 = blockIdx.y * LR_HEADS;
  const int64_t i = blockIdx.z;
  const int H = p.a.heads, R = p.a.rank, RD = p.a.rot, D = R + RD, KL = p.kv.k_ld;
  const int nh = min(LR_HEADS, H - h0);
  float* qs = sm;                   // [LR_HEADS][KL]
  float* acc = qs + LR_HEADS * KL;  // [LR_HEADS][KL]
  pdl_launch_dependents();
  const LatentSpan s = latent_span(p, i, part);
  if ((uint32_t)part >= s.n_parts) return;
  pdl_wait();
  for (int k = tid; k < LR_HEADS * KL; k += LR_THREADS) {
    const int h = k / KL, d = k - h * KL;
    float v = 0.f;
    if (h < nh && d < R) v = p.r.q_lat[i * p.r.q_row + (h0 + h) * p.r.q_head + d];
    if (h < nh && d >= R && d < D) {
      const int e = d - R;
      const int64_t at = s.t * p.r.q.ld + (int64_t)(h0 + h) * (p.a.dim + RD) + p.a.dim + (e & ~1);
      float sn, cs;
      rope_sincos(s.pos, p.a.freq[e / 2], &sn, &cs);
      const float x = latent_q_value(p.r.q, at), y = latent_q_value(p.r.q, at + 1);
      v = e & 1 ? y * cs + x * sn : x * cs - y * sn;
    }
    qs[k] = from_elem(to_elem<E>(v));
    acc[k] = 0.f;
  }
  const E* pool = reinterpret_cast<const E*>(p.kv.base);
  float m = -INFINITY, l = 0.f;  // warp w: of head w
  for (uint32_t k0 = s.k_begin; k0 < s.k_end; k0 += LR_TILE) {
    const int n = (int)min((uint32_t)LR_TILE, s.k_end - k0);
    __syncthreads();
    if (tid < n) {
      uint32_t block = s.table[(k0 + tid) / p.kv.block_size];
      if (block >= p.kv.num_blocks) {
        atomicOr(p.status, DEV_BAD_INDEX);
        block = 0;
      }
      key_at[tid] = p.kv.k_elem(block, 0, (k0 + tid) % p.kv.block_size);
    }
    __syncthreads();
    for (int key = warp; key < n; key += LR_THREADS / 32) {
      const E* row = pool + key_at[key];
      float dot[LR_HEADS] = {0.f, 0.f, 0.f, 0.f};
      for (int c = lane; c < KL / 8; c += 32) {
        float kf[8];
        expand(load_raw(row + c * 8), kf);
#pragma unroll
        for (int h = 0; h < LR_HEADS; ++h)
#pragma unroll
          for (int e = 0; e < 8; ++e) dot[h] = fmaf(qs[h * KL + c * 8 + e], kf[e], dot[h]);
      }
#pragma unroll
      for (int h = 0; h < LR_HEADS; ++h) {
#pragma unroll
        for (int o = 16; o; o >>= 1) dot[h] += __shfl_xor_sync(0xFFFFFFFFu, dot[h], o);
        if (lane == 0) prob[h][key] = dot[h] * p.a.scale;
      }
    }
    __syncthreads();
    {
      const float v = lane < n ? prob[warp][lane] : -INFINITY;
      float top = v;
#pragma unroll
      for (int o = 16; o; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xFFFFFFFFu, top, o));
      top = fmaxf(top, m);
      const float w = expf(v - top), c = expf(m - top);
      float sum = w;
#pragma unroll
      for (int o = 16; o; o >>= 1) sum += __shfl_xor_sync(0xFFFFFFFFu, sum, o);
      l = l * c + sum;
      m = top;
      prob[warp][lane] = w;
      if (lane == 0) corr[warp] = c;
    }
    __syncthreads();
    for (int c = tid; c < R; c += LR_THREADS) {
      float o[LR_HEADS];
#pragma unroll
      for (int h = 0; h < LR_HEADS; ++h) o[h] = acc[h * KL + c] * corr[h];
      for (int key = 0; key < n; ++key) {
        const float v = from_elem(pool[key_at[key] + c]);
#pragma unroll
        for (int h = 0; h < LR_HEADS; ++h) o[h] = fmaf(prob[h][key], v, o[h]);
      }
#pragma unroll
      for (int h = 0; h < LR_HEADS; ++h) acc[h * KL + c] = o[h];
    }
  }
  __syncthreads();
  if (p.parts == 1) {
    if (lane == 0 && warp < nh) {
      const float sink = p.a.sink[h0 + warp], top = fmaxf(m, sink), c = expf(m - top);
      corr[warp] = c / (l * c + expf(sink - top));
    }
    __syncthreads();
    for (int k = tid; k < nh * R; k += LR_THREADS) {
      const int h = k / R, c = k - h * R;
      latent_out<E>(p, i, h0 + h, c, acc[h * KL + c] * corr[h]);
    }
    return;
  }
  float* mine = p.partial + (((size_t)i * H + h0) * p.parts + part) * p.rec;
  const size_t head = (size_t)p.parts * p.rec;
  for (int k = tid; k < nh * R; k += LR_THREADS) {
    const int h = k / R, c = k - h * R;
    mine[h * head + c] = acc[h * KL + c];
  }
  if (lane == 0 && warp < nh) {
    mine[warp * head + p.rec - 4] = m;
    mine[warp * head + p.rec - 3] = l;
  }
}

// ------------------------------------------------- sixteen heads as an mma tile (bf16) ----
// Warp 8 brings the cache rows by tensor map, tiles of 32 keys in panels of 64 columns (128-byte
// swizzle), into a ring of stages. Warps 0-7: for the scores a warp takes 16 of a tile's keys and
// one quarter of the columns; the quarters meet in shared memory, where sixteen threads per head
// form the weights with a running maximum; for weights x values a warp owns every eighth slab of
// the value columns, NVT tiles of 8.
constexpr int LG_WORKERS = 256, LG_THREADS = 288, LG_KEYS = 32, LG_SP = LG_KEYS + 4,
              LG_PS = LG_KEYS + 8;
constexpr int LG_PANEL = LG_KEYS * 128;  // bytes
constexpr int LG_MAX_STAGES = 6;

__device__ __forceinline__ void lg_sync() {
  asm volatile("bar.sync 1, %0;" ::"n"(LG_WORKERS) : "memory");
}
// Row r, 16-byte chunk c (8 columns) of a staged tile.
__device__ __forceinline__ uint32_t lg_addr(uint32_t tile, int r, int c) {
  return tile + (uint32_t)((c >> 3) * LG_PANEL + r * 128 + (((c & 7) ^ (r & 7)) << 4));
}

template <int NVT>
__global__ void __launch_bounds__(LG_THREADS)
    latent_group_kernel(const __grid_constant__ CUtensorMap map, const LatentRowsArgs p) {
  extern __shared__ uint8_t raw[];
  __shared__ uint64_t full[LG_MAX_STAGES], empty[LG_MAX_STAGES];
  __shared__ float corr[16];
  __shared__ volatile int producer_failed, failed;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int part = blockIdx.x, h0 = blockIdx.y * 16;
  const int64_t i = blockIdx.z;
  const KvDenseLayer& kv = p.kv;
  const int H = p.a.heads, R = p.a.rank, RD = p.a.rot, D = R + RD, BS = kv.block_size;
  const int nh = min(16, H - h0);
  const int dp = (D + 15) & ~15, ks = dp + 8, panels = (D + 63) / 64;
  const uint32_t stage_bytes = (uint32_t)panels * LG_PANEL;
  uint8_t* ring = raw + ((1024u - (smem_u32(raw) & 1023u)) & 1023u);
  bf16* Qs = reinterpret_cast<bf16*>(ring + (size_t)p.stages * stage_bytes);  // [16][ks]
  float* Sp = reinterpret_cast<float*>(Qs + 16 * ks);                         // [4][16][LG_SP]
  bf16* Ps = reinterpret_cast<bf16*>(Sp + 4 * 16 * LG_SP);                    // [16][LG_PS]
  float2* turn = reinterpret_cast<float2*>(Ps + 16 * LG_PS);                  // [RD / 2]

  pdl_launch_dependents();
  const LatentSpan s = latent_span(p, i, part);
  if ((uint32_t)part >= s.n_parts) return;
  const int n_tiles = (int)((s.k_end - s.k_begin + LG_KEYS - 1) / LG_KEYS);
  if (tid == 0) {
    for (int k = 0; k < p.stages; ++k) {
      mbar_init(&full[k], 1);
      mbar_init(&empty[k], LG_WORKERS / 32);
    }
    mbar_fence_init();
    producer_failed = failed = 0;
  }
  __syncthreads();

  if (warp == 8) {
    // boxes of at most a page; lane l brings piece l of a tile
    const int box = min(BS, LG_KEYS), pieces = LG_KEYS / box;
    const uint32_t last = (s.k_end - 1) / BS;
    auto page_of = [&](int k) {
      const uint32_t j = s.k_begin + (uint32_t)k * LG_KEYS + (uint32_t)min(lane, pieces - 1) * box;
      // pages past the last key hold none that is seen: the last one stands in for them
      uint32_t b = s.table[min(j / BS, last)];
      if (b >= kv.num_blocks) {
        atomicOr(p.status, DEV_BAD_INDEX);
        b = 0;
      }
      return b;
    };
    bool waited = false;
    int issued = 0;
    uint32_t block = page_of(0);
    for (int k = 0; k < n_tiles; ++k) {
      const int st = k % p.stages;
      const uint32_t next = k + 1 < n_tiles ? page_of(k + 1) : 0u;
      // rows that earlier steps have stored may be asked for before the wait
      if (!waited && !(p.r.early && s.k_begin + (uint32_t)(k + 1) * LG_KEYS <= s.pos)) {
        pdl_wait();
        asm volatile("fence.proxy.async;" ::: "memory");
        waited = true;
      }
      const bool ok =
          mbar_wait_bounded(&empty[st], ((uint32_t)(k / p.stages) & 1u) ^ 1u) && !failed;
      if (!__all_sync(0xFFFFFFFFu, ok)) {
        producer_failed = 1;
        break;
      }
      if (lane == 0) mbar_arrive_expect_tx(&full[st], stage_bytes);
      __syncwarp();
      const int row = (int)((s.k_begin + (uint32_t)k * LG_KEYS) % BS);  // not 0: a page of 64 and more
      if (lane < pieces)
        for (int c = 0; c < panels; ++c)
          tma_load_3d(ring + (size_t)st * stage_bytes + (size_t)c * LG_PANEL + lane * box * 128,
                      &map, c * 64, row, (int)block, &full[st]);
      issued = k + 1;
      block = next;
    }
    // leave only when every copy has landed (bounded)
    if (lane == 0)
      for (int k = max(0, issued - p.stages); k < issued; ++k)
        mbar_wait_bounded(&full[k % p.stages], (uint32_t)(k / p.stages) & 1u);
    return;
  }

  for (int k = tid; k < RD / 2; k += LG_WORKERS)
    rope_sincos(s.pos, p.a.freq[k], &turn[k].x, &turn[k].y);
  for (int k = tid; k < 16 * ks / 8; k += LG_WORKERS)
    reinterpret_cast<uint4*>(Qs)[k] = make_uint4(0u, 0u, 0u, 0u);
  lg_sync();
  pdl_wait();
  {
    const float* ql = p.r.q_lat + i * p.r.q_row + (int64_t)h0 * p.r.q_head;
    if (R % 4 == 0 && p.r.q_head % 4 == 0 && p.r.q_row % 4 == 0) {
      const int r4 = R / 4;
#pragma unroll 8
      for (int k = tid; k < nh * r4; k += LG_WORKERS) {
        const int h = k / r4, d = (k - h * r4) * 4;
        const float4 v = *reinterpret_cast<const float4*>(ql + h * p.r.q_head + d);
        *reinterpret_cast<uint2*>(Qs + h * ks + d) =
            make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
      }
    } else {
      for (int k = tid; k < nh * R; k += LG_WORKERS) {
        const int h = k / R, d = k - h * R;
        Qs[h * ks + d] = to_elem<bf16>(ql[h * p.r.q_head + d]);
      }
    }
    const int r2 = RD / 2;
    for (int k = tid; k < nh * r2; k += LG_WORKERS) {
      const int h = k / r2, e = k - h * r2;
      const int64_t at =
          s.t * p.r.q.ld + (int64_t)(h0 + h) * (p.a.dim + RD) + p.a.dim + 2 * e;
      const float x = latent_q_value(p.r.q, at), y = latent_q_value(p.r.q, at + 1);
      const float2 sc = turn[e];
      Qs[h * ks + R + 2 * e] = to_elem<bf16>(x * sc.y - y * sc.x);
      Qs[h * ks + R + 2 * e + 1] = to_elem<bf16>(y * sc.y + x * sc.x);
    }
  }
  lg_sync();

  float o[NVT][4];
#pragma unroll
  for (int k = 0; k < NVT; ++k) o[k][0] = o[k][1] = o[k][2] = o[k][3] = 0.f;
  const float L2E = 1.44269504088896340736f;
  const float k1 = p.a.scale * L2E;
  float m = -INFINITY, l = 0.f;  // in units of log2; sixteen threads per head, l their own keys'
  const int head = tid >> 4, sub = tid & 15;
  const int nk = dp / 16, quarter = warp >> 1, kb = quarter * nk / 4, ke = (quarter + 1) * nk / 4;
  const int row = lane >> 2;
  const int v0 = warp * NVT * 8;  // first value column of the warp
  const int v_end = (R + 15) & ~15;
  const uint32_t qa = smem_u32(Qs) + (uint32_t)((lane & 15) * ks + (lane >> 4) * 8) * 2;
  const uint32_t pa = smem_u32(Ps) + (uint32_t)((lane & 15) * LG_PS + (lane >> 4) * 8) * 2;
  const int kr = (warp & 1) * 16 + (lane & 7) + ((lane >> 4) << 3);  // key row of the lane's address
  for (int k = 0; k < n_tiles; ++k) {
    const int st = k % p.stages;
    const uint32_t k0 = s.k_begin + (uint32_t)k * LG_KEYS;
    bool ok = false;
    for (uint32_t n = 0; n < (1u << 22) && !ok; ++n) {
      ok = mbar_try_wait(&full[st], (uint32_t)(k / p.stages) & 1u);
      if (!ok && (n & 63u) == 63u && producer_failed) break;
    }
    if (!ok) failed = 1;  // read by all after the next barrier, written by none until then
    const uint32_t tile = smem_u32(ring) + (uint32_t)st * stage_bytes;
    {
      float c[2][4] = {};
#pragma unroll 4
      for (int kk = kb; kk < ke; ++kk) {
        uint32_t a[4], b[4];
        ldm_x4(a, qa + kk * 32);
        ldm_x4(b, lg_addr(tile, kr, kk * 2 + ((lane >> 3) & 1)));
        mma_bf16(c[0], a, b[0], b[1]);
        mma_bf16(c[1], a, b[2], b[3]);
      }
      float* dst = Sp + (quarter * 16 + row) * LG_SP + (warp & 1) * 16 + (lane & 3) * 2;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        *reinterpret_cast<float2*>(dst + nt * 8) = make_float2(c[nt][0], c[nt][1]);
        *reinterpret_cast<float2*>(dst + 8 * LG_SP + nt * 8) = make_float2(c[nt][2], c[nt][3]);
      }
    }
    lg_sync();
    if (failed) break;
    {
      float v[2] = {0.f, 0.f};
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 x = *reinterpret_cast<const float2*>(Sp + (q * 16 + head) * LG_SP + sub * 2);
        v[0] += x.x, v[1] += x.y;
      }
      v[0] = k0 + sub * 2 < s.k_end ? v[0] * k1 : -INFINITY;
      v[1] = k0 + sub * 2 + 1 < s.k_end ? v[1] * k1 : -INFINITY;
      float top = fmaxf(v[0], v[1]);
#pragma unroll
      for (int q = 8; q; q >>= 1) top = fmaxf(top, __shfl_xor_sync(0xFFFFFFFFu, top, q));
      top = fmaxf(top, m);
      const float c = ex2_approx(m - top);
      m = top;
      v[0] = ex2_approx(v[0] - top), v[1] = ex2_approx(v[1] - top);
      l = l * c + v[0] + v[1];
      *reinterpret_cast<uint32_t*>(Ps + head * LG_PS + sub * 2) = pack_bf16(v[0], v[1]);
      if (sub == 0) corr[head] = c;
    }
    lg_sync();
    const float c0 = corr[row], c1 = corr[row + 8];
    uint32_t a[2][4];
    ldm_x4(a[0], pa);
    ldm_x4(a[1], pa + 32);
#pragma unroll
    for (int nt = 0; nt < NVT; nt += 2) {
      if (v0 + nt * 8 < v_end) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          o[nt + e][0] *= c0, o[nt + e][1] *= c0;
          o[nt + e][2] *= c1, o[nt + e][3] *= c1;
        }
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
          uint32_t b[4];
          ldm_x4_t(b, lg_addr(tile, kk * 16 + (lane & 15), v0 / 8 + nt + (lane >> 4)));
          mma_bf16(o[nt], a[kk], b[0], b[1]);
          mma_bf16(o[nt + 1], a[kk], b[2], b[3]);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[st]);
  }
#pragma unroll
  for (int q = 8; q; q >>= 1) l += __shfl_xor_sync(0xFFFFFFFFu, l, q);
  if (failed) {
    if (tid == 0) atomicOr(p.status, DEV_WAIT_TIMEOUT);
    return;
  }
  if (p.parts == 1) {
    lg_sync();  // corr has been read
    if (sub == 0 && head < nh) {
      const float sink = p.a.sink[h0 + head] * L2E, top = fmaxf(m, sink), c = exp2f(m - top);
      corr[head] = c / (l * c + exp2f(sink - top));
    }
    lg_sync();
#pragma unroll
    for (int nt = 0; nt < NVT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = row + (e >> 1) * 8, c = v0 + nt * 8 + (lane & 3) * 2 + (e & 1);
        if (h < nh && c < R) latent_out<bf16>(p, i, h0 + h, c, o[nt][e] * corr[h]);
      }
    return;
  }
  float* mine = p.partial + (((size_t)i * H + h0) * p.parts + part) * p.rec;
  const size_t step = (size_t)p.parts * p.rec;
#pragma unroll
  for (int nt = 0; nt < NVT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int h = row + (e >> 1) * 8, c = v0 + nt * 8 + (lane & 3) * 2;
      // an odd last column takes the place of the pad behind it along
      if (h < nh && c < R)
        *reinterpret_cast<float2*>(mine + h * step + c) = make_float2(o[nt][e], o[nt][e + 1]);
    }
  if (sub == 0 && head < nh) {
    mine[head * step + p.rec - 4] = m * (1.0f / L2E);
    mine[head * step + p.rec - 3] = l;
  }
}

template <int NVT>
static int32_t group_launch(kanso_cuda_ctx* ctx, dim3 grid, size_t smem, const CUtensorMap& map,
                            const LatentRowsArgs& p) {
  int32_t st = allow_max_smem(ctx, (const void*)latent_group_kernel<NVT>);
  if (st) return st;
  const cudaError_t e =
      launch_dependent(ctx, latent_group_kernel<NVT>, grid, dim3(LG_THREADS), smem, map, p);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "latent attention launch");
  return after_launch(ctx, "latent_group");
}

// Stages of the tile form's ring and its shared memory; 0 stages: it does not fit.
static int group_stages(const LatentAttn& a, uint32_t k_dim, size_t* smem) {
  const size_t stage = (size_t)((k_dim + 63) / 64) * LG_PANEL;
  const size_t rest = 1024 + (size_t)16 * (((k_dim + 15u) & ~15u) + 8) * 2 + 4 * 16 * LG_SP * 4 +
                      16 * LG_PS * 2 + (size_t)a.rot * 4;
  // two CTAs per SM where two stages leave room for it: one's barriers are the other's work
  const size_t room = 2 * stage + rest <= 110 * 1024 ? 110 * 1024 : 222 * 1024;
  int n = LG_MAX_STAGES;
  while (n > 0 && n * stage + rest > room) --n;
  *smem = n * stage + rest;
  return n >= 2 ? n : 0;
}

int32_t launch_latent_attn_rows(kanso_cuda_ctx* ctx, int32_t compute, const LatentAttn& a,
                                const KvDenseLayer& kv, const LatentRows& r, int path,
                                bool* handled) {
  *handled = true;
  if (r.n > 65535)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "attention: %lld rows in one launch", (long long)r.n);
  LatentRowsArgs p;
  p.a = a;
  p.kv = kv;
  p.r = r;
  p.partial = nullptr;
  p.status = ctx->dev_status;
  size_t smem = 0;
  p.stages = group_stages(a, kv.k_dim, &smem);
  const uint32_t bs = kv.block_size;
  bool group = path != 1 && compute == KANSO_COMPUTE_BF16 && a.rank <= 1024 && p.stages &&
               (bs == 8 || bs == 16 || bs % 32 == 0) && kv.num_blocks < (1u << 31);
  CUtensorMap map;
  if (group) {
    TmEncodeFn encode = tm_encoder();
    group = encode && tm_map3(encode, kv.base, kv.k_ld, bs, kv.num_blocks, kv.k_ld, kv.rec_elems,
                              std::min<uint32_t>(bs, LG_KEYS), 1, &map);
  }
  if (path == 2 && !group) {
    *handled = false;
    return KANSO_OK;
  }
  p.tile = group ? LG_KEYS : LR_TILE;
  p.rec = ((a.rank + 3u) & ~3u) + 4;
  const uint32_t HB = group ? (a.heads + 15) / 16 : (a.heads + LR_HEADS - 1) / LR_HEADS;
  const uint32_t tiles = std::max(1u, (r.max_keys + p.tile - 1) / p.tile);
  const uint64_t ctas = (uint64_t)r.n * HB;
  // Shares of the keys. The tile form: the split with the shortest run of waves, a wave being a
  // share's tiles and a few tiles' worth of fixed work; the plain form: four CTAs per SM.
  uint32_t parts = 1;
  if (group) {
    const uint64_t per_sm = std::max<uint64_t>(
        1, std::min<uint64_t>(4, (uint64_t)ctx->smem_per_sm / (smem + 1200)));
    const uint64_t resident = (uint64_t)ctx->sm_count * per_sm;
    uint64_t best = ~0ull;
    for (uint32_t n = 1; n <= std::min(tiles, 256u); ++n) {
      const uint64_t cost =
          (ctas * n + resident - 1) / resident * ((tiles + n - 1) / n + 6) + (n > 1 ? 6 : 0);
      if (cost < best) {
        best = cost;
        parts = n;
      }
    }
  } else {
    parts = (uint32_t)std::min<uint64_t>(std::min(tiles, 256u),
                                         std::max<uint64_t>(1, 4ull * ctx->sm_count / ctas));
  }
  const uint32_t per = (tiles + parts - 1) / parts;
  p.parts = (tiles + per - 1) / per;
  if (p.parts > 1) {
    p.partial = (float*)ctx_scratch(ctx, (size_t)r.n * a.heads * p.parts * p.rec * 4);
    if (!p.partial) return KANSO_ERR_DEVICE;
  }
  const dim3 grid(p.parts, HB, (unsigned)r.n);
  int32_t st;
  if (group) {
    st = a.rank <= 128   ? group_launch<2>(ctx, grid, smem, map, p)
         : a.rank <= 256 ? group_launch<4>(ctx, grid, smem, map, p)
         : a.rank <= 512 ? group_launch<8>(ctx, grid, smem, map, p)
                         : group_launch<16>(ctx, grid, smem, map, p);
    if (st) return st;
  } else {
    smem = (size_t)2 * LR_HEADS * kv.k_ld * 4;
    if (smem > 200 * 1024)
      return fail(ctx, KANSO_ERR_UNSUPPORTED, "latent attention: cache rows of %u columns",
                  kv.k_dim);
    auto kern =
        compute == KANSO_COMPUTE_BF16 ? latent_rows_kernel<bf16> : latent_rows_kernel<float>;
    if ((st = allow_max_smem(ctx, (const void*)kern))) return st;
    const cudaError_t e = launch_dependent(ctx, kern, grid, dim3(LR_THREADS), smem, p);
    if (e != cudaSuccess) return cuda_fail(ctx, e, "latent attention launch");
    if ((st = after_launch(ctx, "latent_rows"))) return st;
  }
  if (p.parts == 1) return KANSO_OK;
  auto merge =
      compute == KANSO_COMPUTE_BF16 ? latent_merge_kernel<bf16> : latent_merge_kernel<float>;
  const uint32_t slabs = (a.rank + LM_COLS - 1) / LM_COLS;
  const dim3 mgrid(a.heads, (unsigned)r.n,
                   (uint64_t)a.heads * r.n * 2 > (uint64_t)ctx->sm_count * 8 ? 1 : slabs);
  const cudaError_t e =
      launch_dependent(ctx, merge, mgrid, dim3(LM_THREADS), (size_t)p.parts * 8, p);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "latent merge launch");
  return after_launch(ctx, "latent_merge");
}

}  // namespace kanso
