// Softmax attention on cached latents, for decoding and short portions. A token's cache row is
// [c | k_rot]; with the query's unrotated part taken through the transposed key projection
// beforehand (q_lat = W_uk^T q) and the value projection applied afterwards, every head reads the
// same rows:
//
//   s = scale * (q_lat . c_j + q_rot . k_rot_j),  0 <= j <= i
//   out = sum_j exp(s_j) c_j / (sum_j exp(s_j) + exp(sink))
//
// latent_rows: four heads per CTA, any size, f32 and (sizes beyond the other) bfloat16.
// latent_group: bfloat16, sixteen heads as the rows of an mma tile, 64 keys at a time; a staged row
// serves as key and as value. A row's keys may be shared out over several CTAs: partial sums with
// their maxima are merged in order by the CTA that arrives last.
#include <algorithm>
#include <cmath>

#include "dense.cuh"
#include "warp_mma.cuh"

namespace kanso {

struct LatentRowsArgs {
  LatentAttn a;
  KvDenseLayer kv;
  LatentRows r;
  float* partial;   // [n][heads][parts][rank + 2]: sums, maximum, denominator
  uint32_t* tickets;
  uint32_t parts, tile;
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
// The shares of heads [h0, h0 + nh) of row i, and the store of the result. All threads.
template <typename E>
__device__ __forceinline__ void latent_merge(const LatentRowsArgs& p, int64_t i, int h0, int nh,
                                             uint32_t n_parts, float* coef) {
  const int R = p.a.rank;
  const size_t rec = (size_t)R + 2;
  const float* src = p.partial + ((size_t)i * p.a.heads + h0) * p.parts * rec;
  for (int h = threadIdx.x; h < nh; h += blockDim.x) {
    const float* m = src + (size_t)h * p.parts * rec + R;
    const float sink = p.a.sink[h0 + h];
    float top = sink, den = 0.f;
    for (uint32_t k = 0; k < n_parts; ++k) top = fmaxf(top, __ldcg(m + k * rec));
    for (uint32_t k = 0; k < n_parts; ++k)
      den += __ldcg(m + k * rec + 1) * expf(__ldcg(m + k * rec) - top);
    coef[2 * h] = top;
    coef[2 * h + 1] = 1.0f / (den + expf(sink - top));
  }
  __syncthreads();
  for (int k = threadIdx.x; k < nh * R; k += blockDim.x) {
    const int h = k / R, c = k - h * R;
    const float* o = src + (size_t)h * p.parts * rec;
    float v = 0.f;
    for (uint32_t s = 0; s < n_parts; ++s)
      v += __ldcg(o + s * rec + c) * expf(__ldcg(o + s * rec + R) - coef[2 * h]);
    v *= coef[2 * h + 1];
    const int64_t at = i * p.r.out_row + (h0 + h) * p.r.out_head + c;
    if (p.r.out_f32)
      static_cast<float*>(p.r.out)[at] = v;
    else
      static_cast<E*>(p.r.out)[at] = to_elem<E>(v);
  }
}

// ------------------------------------------------------------------------ any size ----
constexpr int LR_THREADS = 128, LR_HEADS = 4, LR_TILE = 32;

template <typename E>
__global__ void __launch_bounds__(LR_THREADS) latent_rows_kernel(const LatentRowsArgs p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float prob[LR_HEADS][LR_TILE], corr[LR_HEADS], coef[2 * LR_HEADS];
  __shared__ size_t key_at[LR_TILE];
  __shared__ uint32_t ticket;
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
  if (s.n_parts == 1) {
    if (lane == 0 && warp < nh) {
      const float sink = p.a.sink[h0 + warp], top = fmaxf(m, sink), c = expf(m - top);
      corr[warp] = c / (l * c + expf(sink - top));
    }
    __syncthreads();
    for (int k = tid; k < nh * R; k += LR_THREADS) {
      const int h = k / R, c = k - h * R;
      const float v = acc[h * KL + c] * corr[h];
      const int64_t at = i * p.r.out_row + (h0 + h) * p.r.out_head + c;
      if (p.r.out_f32)
        static_cast<float*>(p.r.out)[at] = v;
      else
        static_cast<E*>(p.r.out)[at] = to_elem<E>(v);
    }
    return;
  }
  const size_t rec = (size_t)R + 2;
  float* mine = p.partial + ((size_t)i * H + h0) * p.parts * rec + part * rec;
  for (int k = tid; k < nh * R; k += LR_THREADS) {
    const int h = k / R, c = k - h * R;
    mine[(size_t)h * p.parts * rec + c] = acc[h * KL + c];
  }
  if (lane == 0 && warp < nh) {
    mine[(size_t)warp * p.parts * rec + R] = m;
    mine[(size_t)warp * p.parts * rec + R + 1] = l;
  }
  __threadfence();
  __syncthreads();
  uint32_t* tk = &p.tickets[i * gridDim.y + blockIdx.y];
  if (tid == 0) ticket = atomicAdd(tk, 1u);
  __syncthreads();
  if (ticket != s.n_parts - 1) return;
  __threadfence();
  latent_merge<E>(p, i, h0, nh, s.n_parts, coef);
  if (tid == 0) *tk = 0;
}

// ------------------------------------------------- sixteen heads as an mma tile (bf16) ----
// Eight warps. Scores: warp w takes 16 of a tile's 64 keys and one half of the columns; the halves
// meet in shared memory, where sixteen threads per head form the weights with a running
// maximum. Weights x values: warp w owns every eighth slab of the value columns, NVT tiles of 8.
constexpr int LG_THREADS = 256, LG_KEYS = 64, LG_SP = LG_KEYS + 4, LG_PS = LG_KEYS + 8;

template <int NVT>
__global__ void __launch_bounds__(LG_THREADS) latent_group_kernel(const LatentRowsArgs p) {
  extern __shared__ __align__(16) uint8_t sm_raw[];
  __shared__ float corr[16], den[16], top_s[16], coef[32];
  __shared__ uint32_t ticket;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int part = blockIdx.x, h0 = blockIdx.y * 16;
  const int64_t i = blockIdx.z;
  const KvDenseLayer& kv = p.kv;
  const int H = p.a.heads, R = p.a.rank, RD = p.a.rot, D = R + RD, KL = kv.k_ld, BS = kv.block_size;
  const int nh = min(16, H - h0);
  const int dp = (D + 15) & ~15, ks = dp + 8;
  bf16* Qs = reinterpret_cast<bf16*>(sm_raw);             // [16][ks]
  bf16* Ks = Qs + 16 * ks;                                // two tiles [64][ks]
  float* Sp = reinterpret_cast<float*>(Ks + 2 * LG_KEYS * ks);  // [2][16][LG_SP]
  bf16* Ps = reinterpret_cast<bf16*>(Sp + 2 * 16 * LG_SP);      // [16][LG_PS]
  float2* turn = reinterpret_cast<float2*>(Ps + 16 * LG_PS);    // [RD / 2]

  pdl_launch_dependents();
  const LatentSpan s = latent_span(p, i, part);
  if ((uint32_t)part >= s.n_parts) return;
  const bf16* pool = reinterpret_cast<const bf16*>(kv.base);
  const int kc = dp / 8, kl = KL / 8;
  // 16-byte pieces of a tile: thread tid takes piece (tid % 4) + 4 * n of row tid / 4
  auto fetch = [&](uint32_t k0, int buf) {
    const int r = tid >> 2;
    const uint32_t j = k0 + r;
    bool in = j < s.k_end;
    size_t at = 0;
    if (in) {
      const uint32_t block = s.table[j / BS];
      if (block < kv.num_blocks) {
        at = kv.k_elem(block, 0, j % BS);
      } else {
        atomicOr(p.status, DEV_BAD_INDEX);
        in = false;
      }
    }
    bf16* dst = Ks + (size_t)(buf * LG_KEYS + r) * ks;
    for (int c = tid & 3; c < kc; c += 4) {
      const bool ok = in && c < kl;
      cp_async16(dst + c * 8, ok ? pool + at + c * 8 : pool, ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // the first tile may be asked for before the wait when the step's own row is not in it
  const bool early = p.r.early && s.k_begin + LG_KEYS <= s.pos;
  if (early) fetch(s.k_begin, 0);
  for (int k = tid; k < RD / 2; k += LG_THREADS) rope_sincos(s.pos, p.a.freq[k], &turn[k].x, &turn[k].y);
  for (int k = tid; k < 16 * ks / 8; k += LG_THREADS)
    reinterpret_cast<uint4*>(Qs)[k] = make_uint4(0u, 0u, 0u, 0u);
  __syncthreads();
  pdl_wait();
  if (!early) fetch(s.k_begin, 0);
  {
    const float* ql = p.r.q_lat + i * p.r.q_row + (int64_t)h0 * p.r.q_head;
    if (R % 4 == 0 && p.r.q_head % 4 == 0 && p.r.q_row % 4 == 0) {
      const int r4 = R / 4;
#pragma unroll 4
      for (int k = tid; k < nh * r4; k += LG_THREADS) {
        const int h = k / r4, d = (k - h * r4) * 4;
        const float4 v = *reinterpret_cast<const float4*>(ql + h * p.r.q_head + d);
        *reinterpret_cast<uint2*>(Qs + h * ks + d) =
            make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
      }
    } else {
      for (int k = tid; k < nh * R; k += LG_THREADS) {
        const int h = k / R, d = k - h * R;
        Qs[h * ks + d] = to_elem<bf16>(ql[h * p.r.q_head + d]);
      }
    }
    const int r2 = RD / 2;
    for (int k = tid; k < nh * r2; k += LG_THREADS) {
      const int h = k / r2, e = k - h * r2;
      const int64_t at =
          s.t * p.r.q.ld + (int64_t)(h0 + h) * (p.a.dim + RD) + p.a.dim + 2 * e;
      const float x = latent_q_value(p.r.q, at), y = latent_q_value(p.r.q, at + 1);
      const float2 sc = turn[e];
      Qs[h * ks + R + 2 * e] = to_elem<bf16>(x * sc.y - y * sc.x);
      Qs[h * ks + R + 2 * e + 1] = to_elem<bf16>(y * sc.y + x * sc.x);
    }
  }

  float o[NVT][4];
#pragma unroll
  for (int k = 0; k < NVT; ++k) o[k][0] = o[k][1] = o[k][2] = o[k][3] = 0.f;
  const float L2E = 1.44269504088896340736f;
  const float k1 = p.a.scale * L2E;
  float m = -INFINITY, l = 0.f;  // in units of log2; sixteen threads per head, l their own keys'
  const int head = tid >> 4, sub = tid & 15;
  const int nk = dp / 16, half = warp >> 2, kb = half ? (nk + 1) / 2 : 0,
            ke = half ? nk : (nk + 1) / 2;
  const int row = lane >> 2;
  const int v0 = warp * NVT * 8;  // first value column of the warp
  const int v_end = (R + 15) & ~15;
  const uint32_t qa = smem_u32(Qs) + (uint32_t)((lane & 15) * ks + (lane >> 4) * 8) * 2;
  const uint32_t pa = smem_u32(Ps) + (uint32_t)((lane & 15) * LG_PS + (lane >> 4) * 8) * 2;
  int buf = 0;
  for (uint32_t k0 = s.k_begin; k0 < s.k_end; k0 += LG_KEYS, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this tile has landed, nobody reads the other buffer
    if (k0 + LG_KEYS < s.k_end) fetch(k0 + LG_KEYS, buf ^ 1);
    const bf16* Kt = Ks + (size_t)buf * LG_KEYS * ks;
    {
      float c[2][4] = {};
      const uint32_t ka = smem_u32(Kt) +
                          (uint32_t)(((warp & 3) * 16 + (lane & 7) + ((lane >> 4) << 3)) * ks +
                                     ((lane >> 3) & 1) * 8) * 2;
#pragma unroll 4
      for (int kk = kb; kk < ke; ++kk) {
        uint32_t a[4], b[4];
        ldm_x4(a, qa + kk * 32);
        ldm_x4(b, ka + kk * 32);
        mma_bf16(c[0], a, b[0], b[1]);
        mma_bf16(c[1], a, b[2], b[3]);
      }
      float* dst = Sp + (half * 16 + row) * LG_SP + (warp & 3) * 16 + (lane & 3) * 2;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        *reinterpret_cast<float2*>(dst + nt * 8) = make_float2(c[nt][0], c[nt][1]);
        *reinterpret_cast<float2*>(dst + 8 * LG_SP + nt * 8) = make_float2(c[nt][2], c[nt][3]);
      }
    }
    __syncthreads();
    {
      const float4 x = *reinterpret_cast<const float4*>(Sp + head * LG_SP + sub * 4);
      const float4 y = *reinterpret_cast<const float4*>(Sp + (16 + head) * LG_SP + sub * 4);
      float v[4] = {(x.x + y.x) * k1, (x.y + y.y) * k1, (x.z + y.z) * k1, (x.w + y.w) * k1};
      float top = -INFINITY;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (k0 + sub * 4 + e >= s.k_end) v[e] = -INFINITY;
        top = fmaxf(top, v[e]);
      }
#pragma unroll
      for (int q = 8; q; q >>= 1) top = fmaxf(top, __shfl_xor_sync(0xFFFFFFFFu, top, q));
      top = fmaxf(top, m);
      const float c = ex2_approx(m - top);
      m = top;
      l *= c;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[e] = ex2_approx(v[e] - top);
        l += v[e];
      }
      *reinterpret_cast<uint2*>(Ps + head * LG_PS + sub * 4) =
          make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
      if (sub == 0) corr[head] = c;
    }
    __syncthreads();
    const float c0 = corr[row], c1 = corr[row + 8];
    uint32_t a[4][4];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) ldm_x4(a[kk], pa + kk * 32);
    const uint32_t va = smem_u32(Kt) + (uint32_t)((lane & 15) * ks + (lane >> 4) * 8 + v0) * 2;
#pragma unroll
    for (int nt = 0; nt < NVT; nt += 2) {
      if (v0 + nt * 8 < v_end) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          o[nt + e][0] *= c0, o[nt + e][1] *= c0;
          o[nt + e][2] *= c1, o[nt + e][3] *= c1;
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          uint32_t b[4];
          ldm_x4_t(b, va + (uint32_t)(kk * 16 * ks + nt * 8) * 2);
          mma_bf16(o[nt], a[kk], b[0], b[1]);
          mma_bf16(o[nt + 1], a[kk], b[2], b[3]);
        }
      }
    }
  }
#pragma unroll
  for (int q = 8; q; q >>= 1) l += __shfl_xor_sync(0xFFFFFFFFu, l, q);
  __syncthreads();  // corr has been read
  if (sub == 0) {
    top_s[head] = m * (1.0f / L2E);
    den[head] = l;
    if (head < nh) {
      const float sink = p.a.sink[h0 + head] * L2E, top = fmaxf(m, sink), c = exp2f(m - top);
      corr[head] = c / (l * c + exp2f(sink - top));
    }
  }
  __syncthreads();
  if (s.n_parts == 1) {
#pragma unroll
    for (int nt = 0; nt < NVT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int h = row + (e >> 1) * 8, c = v0 + nt * 8 + (lane & 3) * 2;
        if (h >= nh || c >= R) continue;
        const int64_t at = i * p.r.out_row + (h0 + h) * p.r.out_head + c;
        const float x = o[nt][e] * corr[h], y = o[nt][e + 1] * corr[h];
        if (p.r.out_f32) {
          float* dst = static_cast<float*>(p.r.out) + at;
          dst[0] = x;
          if (c + 1 < R) dst[1] = y;
        } else {
          bf16* dst = static_cast<bf16*>(p.r.out) + at;
          dst[0] = to_elem<bf16>(x);
          if (c + 1 < R) dst[1] = to_elem<bf16>(y);
        }
      }
    return;
  }
  const size_t rec = (size_t)R + 2;
  float* mine = p.partial + ((size_t)i * H + h0) * p.parts * rec + part * rec;
#pragma unroll
  for (int nt = 0; nt < NVT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = row + (e >> 1) * 8, c = v0 + nt * 8 + (lane & 3) * 2 + (e & 1);
      if (h < nh && c < R) mine[(size_t)h * p.parts * rec + c] = o[nt][e];
    }
  if (tid < nh) {
    mine[(size_t)tid * p.parts * rec + R] = top_s[tid];
    mine[(size_t)tid * p.parts * rec + R + 1] = den[tid];
  }
  __threadfence();
  __syncthreads();
  uint32_t* tk = &p.tickets[i * gridDim.y + blockIdx.y];
  if (tid == 0) ticket = atomicAdd(tk, 1u);
  __syncthreads();
  if (ticket != s.n_parts - 1) return;
  __threadfence();
  latent_merge<bf16>(p, i, h0, nh, s.n_parts, coef);
  if (tid == 0) *tk = 0;
}

template <int NVT>
static int32_t group_launch(kanso_cuda_ctx* ctx, dim3 grid, size_t smem, const LatentRowsArgs& p) {
  int32_t st = allow_max_smem(ctx, (const void*)latent_group_kernel<NVT>);
  if (st) return st;
  const cudaError_t e =
      launch_dependent(ctx, latent_group_kernel<NVT>, grid, dim3(LG_THREADS), smem, p);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "latent attention launch");
  return after_launch(ctx, "latent_group");
}

int32_t launch_latent_attn_rows(kanso_cuda_ctx* ctx, int32_t compute, const LatentAttn& a,
                                const KvDenseLayer& kv, const LatentRows& r, int path,
                                bool* handled) {
  *handled = true;
  if (r.n > 65535)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "attention: %lld rows in one launch", (long long)r.n);
  const int dp = (int)((kv.k_dim + 15u) & ~15u), ks = dp + 8;
  const size_t gsmem = ((size_t)16 * ks + 2 * (size_t)LG_KEYS * ks) * 2 + 2 * 16 * LG_SP * 4 +
                       16 * LG_PS * 2 + (size_t)a.rot * 4;
  const bool fits = compute == KANSO_COMPUTE_BF16 && a.rank <= 1024 && gsmem <= 224 * 1024;
  if (path == 2 && !fits) {
    *handled = false;
    return KANSO_OK;
  }
  const bool group = fits && path != 1;
  LatentRowsArgs p;
  p.a = a;
  p.kv = kv;
  p.r = r;
  p.partial = nullptr;
  p.tickets = ctx->pa_tickets;
  p.tile = group ? LG_KEYS : LR_TILE;
  p.status = ctx->dev_status;
  const uint32_t HB = group ? (a.heads + 15) / 16 : (a.heads + LR_HEADS - 1) / LR_HEADS;
  const uint32_t tiles = std::max(1u, (r.max_keys + p.tile - 1) / p.tile);
  const uint64_t ctas = (uint64_t)r.n * HB;
  uint32_t parts = 1;
  if (ctas <= kanso_cuda_ctx::kPaTickets) {
    if (group) {
      // the split with the shortest run of waves, a wave being a share's tiles and about two tiles'
      // worth of fixed work
      const uint64_t per_sm = std::max<uint64_t>(
          1, std::min<uint64_t>(4, (uint64_t)ctx->smem_per_sm / (gsmem + 2048)));
      const uint64_t resident = (uint64_t)ctx->sm_count * per_sm;
      uint64_t best = ~0ull;
      for (uint32_t n = 1; n <= tiles; ++n) {
        const uint64_t cost = (ctas * n + resident - 1) / resident * ((tiles + n - 1) / n + 2);
        if (cost < best) {
          best = cost;
          parts = n;
        }
      }
    } else {
      parts = (uint32_t)std::min<uint64_t>(
          tiles, std::max<uint64_t>(1, 4ull * ctx->sm_count / ctas));
    }
  }
  const uint32_t per = (tiles + parts - 1) / parts;
  p.parts = (tiles + per - 1) / per;
  if (p.parts > 1) {
    p.partial = (float*)ctx_scratch(ctx, (size_t)r.n * a.heads * p.parts * (a.rank + 2) * 4);
    if (!p.partial) return KANSO_ERR_DEVICE;
  }
  const dim3 grid(p.parts, HB, (unsigned)r.n);
  if (group) {
    if (a.rank <= 128) return group_launch<2>(ctx, grid, gsmem, p);
    if (a.rank <= 256) return group_launch<4>(ctx, grid, gsmem, p);
    if (a.rank <= 512) return group_launch<8>(ctx, grid, gsmem, p);
    return group_launch<16>(ctx, grid, gsmem, p);
  }
  const size_t smem = (size_t)2 * LR_HEADS * kv.k_ld * 4;
  if (smem > 200 * 1024)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "latent attention: cache rows of %u columns", kv.k_dim);
  auto kern = compute == KANSO_COMPUTE_BF16 ? latent_rows_kernel<bf16> : latent_rows_kernel<float>;
  int32_t st = allow_max_smem(ctx, (const void*)kern);
  if (st) return st;
  const cudaError_t e = launch_dependent(ctx, kern, grid, dim3(LR_THREADS), smem, p);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "latent attention launch");
  return after_launch(ctx, "latent_rows");
}

}  // namespace kanso
