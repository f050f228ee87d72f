// Attention over a paged pool whose weights are sigmoids of the scores instead of a softmax:
//
//   s = cap * tanh(scale * q.k / cap)            (cap 0: s = scale * q.k)
//   w = sigmoid(s + pb[h] - r1[h] * ln(1 + r2[h] * d)),  d = i - j,  0 <= d < window
//   out_i = sum_j w * v_j
//
// There is no normalisation over keys, so partial sums over any split of the keys simply add: no
// running maximum and no rescaling. The head's constant and its distance term come from one
// table per layer, bias[h][d] (distances beyond the table are computed).
//
// sigmoid_rows: one CTA per (share of the keys, kv head, query row) for all query heads of the
// group, any size, f32 and (sizes beyond the others) bfloat16. sigmoid_group: the bfloat16 form
// of it on mma tiles, for decoding and short portions. In the decode step both also normalise
// the row's q and k (each over its whole projection) and store the new k and v.
// sigmoid_tiles: bfloat16 tiles of 64 query rows x 64 keys for prompts.
#include <algorithm>
#include <cmath>

#include "dense.cuh"
#include "warp_mma.cuh"

namespace kanso {

template <bool FAST>
__device__ __forceinline__ float cap_score(float s, float cap) {
  if (cap == 0.f) return s;
  if (FAST) return cap - 2.f * cap * __fdividef(1.f, 1.f + __expf(2.f * s / cap));
  return cap * tanhf(s / cap);
}
template <bool FAST>
__device__ __forceinline__ float sigmoidf(float z) {
  if (FAST) return __fdividef(1.f, 1.f + __expf(-z));
  return 1.f / (1.f + expf(-z));
}
__device__ __forceinline__ float bias_at(const SigmoidAttn& a, int h, uint32_t d) {
  if (d < a.bias_len) return a.bias[(size_t)h * a.bias_len + d];
  return a.pb[h] - a.r1[h] * log1pf(a.r2[h] * (float)d);
}

// ------------------------------------------------------------------ one query row per CTA ----
constexpr int SR_THREADS = 128;
constexpr int SR_TILE = 64;   // keys per trip
constexpr int SR_HEADS = 4;   // query heads per pass over a value row

struct RowsArgs {
  SigmoidAttn a;
  KvDenseLayer kv;
  RowMap map;
  const void* q;   // [T][heads][k_ld], or nullptr: fused
  QkvSource s;     // fused: the rows' raw q, k, v
  void* out;
  int64_t out_ld;
  float* partial;  // [T][heads][parts][v_dim]
  uint32_t* tickets;
  uint32_t parts;
  int out_f32;
  int* status;
};

template <typename E>
__global__ void __launch_bounds__(SR_THREADS) sigmoid_rows_kernel(const RowsArgs p) {
  constexpr bool FAST = sizeof(E) == 2;
  extern __shared__ __align__(16) uint8_t sm_raw[];
  __shared__ float red[32];
  __shared__ uint32_t ticket;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int part = blockIdx.x, g = blockIdx.y;
  const int64_t t = blockIdx.z;
  const KvDenseLayer& kv = p.kv;
  const int G = kv.kv_heads, H = p.a.heads, HG = H / G;
  const int D = kv.k_dim, DV = kv.v_dim, KL = kv.k_ld, VL = kv.v_ld, BS = kv.block_size;

  float* qs = reinterpret_cast<float*>(sm_raw);           // [HG][KL]
  float* ws = qs + HG * KL;                                // [HG][SR_TILE]
  float* acc_s = ws + HG * SR_TILE;                        // [HG][VL]
  float* redv = acc_s + HG * VL;                           // [groups][SR_HEADS][VL]
  const int vchunks = VL / 8;
  const int kgroups = max(1, min(SR_THREADS / vchunks, 16));
  E* newk = reinterpret_cast<E*>(redv + (size_t)kgroups * SR_HEADS * VL);  // [KL]
  E* newv = newk + KL;                                     // [VL]

  pdl_launch_dependents();
  // positions and tables are step inputs, written before the step's first kernel
  const uint32_t pos = p.map.positions[t];
  const uint32_t seq = p.map.row_seq ? p.map.row_seq[t] : (uint32_t)t;
  const uint32_t* table = p.map.tables + (size_t)seq * p.map.max_blocks;
  const uint32_t lo = p.a.window && pos + 1 > p.a.window ? pos + 1 - p.a.window : 0;
  const uint32_t n_keys = pos + 1 - lo;
  const uint32_t n_tiles = (n_keys + SR_TILE - 1) / SR_TILE;
  const uint32_t per = (n_tiles + p.parts - 1) / p.parts;      // tiles per share
  const uint32_t n_parts = (n_tiles + per - 1) / per;          // shares that have keys
  if ((uint32_t)part >= n_parts) return;
  const uint32_t k_begin = lo + part * per * SR_TILE;
  const uint32_t k_end = min(pos + 1, k_begin + per * SR_TILE);
  const bool fused = p.q == nullptr;
  const bool owns_new = fused && k_end == pos + 1;
  pdl_wait();

  if (!fused) {
    const E* q = static_cast<const E*>(p.q) + ((size_t)t * H + (size_t)g * HG) * KL;
    for (int i = tid; i < HG * KL; i += SR_THREADS) qs[i] = from_elem(q[i]);
  } else {
    const int nq = H * D, nk = G * D;
    const float* src = p.s.qkv + t * (int64_t)(nq + nk + G * DV);
    auto value = [&](int i) {
      float v = src[i];
      for (int r = 1; r < p.s.parts; ++r) v += src[r * p.s.part_stride + i];
      return v;
    };
    float ss = 0.f;
    for (int i = tid; i < nq; i += SR_THREADS) {
      const float v = value(i);
      ss += v * v;
    }
    ss = block_sum(ss, red);
    float inv = 1.0f / sqrtf(ss / (float)nq + p.s.eps);
    for (int i = tid; i < HG * KL; i += SR_THREADS) {
      const int hh = i / KL, d = i - hh * KL, c = (g * HG + hh) * D + d;
      // the same rounding as the stored form of a prompt's q
      qs[i] = d < D ? from_elem(to_elem<E>(value(c) * inv * p.s.q_norm[c])) : 0.f;
    }
    if (owns_new) {
      ss = 0.f;
      for (int i = tid; i < nk; i += SR_THREADS) {
        const float v = value(nq + i);
        ss += v * v;
      }
      ss = block_sum(ss, red);
      inv = 1.0f / sqrtf(ss / (float)nk + p.s.eps);
      const uint32_t place = pos / BS;
      uint32_t block = kv.num_blocks;
      if (place < p.map.max_blocks) block = table[place];
      const bool ok = block < kv.num_blocks;
      if (!ok && tid == 0) atomicOr(p.status, DEV_BAD_INDEX);
      E* pool = reinterpret_cast<E*>(kv.base);
      for (int d = tid; d < KL; d += SR_THREADS) {
        const E v = to_elem<E>(
            d < D ? value(nq + g * D + d) * inv * p.s.k_norm[g * D + d] : 0.f);
        newk[d] = v;
        if (ok) pool[kv.k_elem(block, g, pos % BS) + d] = v;
      }
      for (int d = tid; d < VL; d += SR_THREADS) {
        const E v = to_elem<E>(d < DV ? value(nq + nk + g * DV + d) : 0.f);
        newv[d] = v;
        if (ok) pool[kv.v_elem(block, g, pos % BS) + d] = v;
      }
    }
  }
  for (int i = tid; i < HG * VL; i += SR_THREADS) acc_s[i] = 0.f;
  __syncthreads();

  const E* pool = reinterpret_cast<const E*>(kv.base);
  const int kchunks = KL / 8;
  int lpk = 1;  // lanes that share a key
  while (lpk < kchunks && lpk < 32) lpk *= 2;
  const int kpw = 32 / lpk;  // keys per warp and trip
  const int kl = lane / lpk, cl = lane % lpk;
  const int vc = tid % vchunks, kg = tid / vchunks;

  for (uint32_t k0 = k_begin; k0 < k_end; k0 += SR_TILE) {
    const int n = (int)min((uint32_t)SR_TILE, k_end - k0);
    // raw dot products
    for (int kb = warp * kpw; kb < n; kb += (SR_THREADS / 32) * kpw) {
      const int key = kb + kl;
      const bool in = key < n;
      const uint32_t j = k0 + (in ? key : 0);
      const E* kr;
      if (owns_new && j == pos) {
        kr = newk;
      } else {
        uint32_t block = table[j / BS];
        if (block >= kv.num_blocks) {
          atomicOr(p.status, DEV_BAD_INDEX);
          block = 0;
        }
        kr = pool + kv.k_elem(block, g, j % BS);
      }
      for (int h0 = 0; h0 < HG; h0 += SR_HEADS) {
        float dot[SR_HEADS] = {0.f, 0.f, 0.f, 0.f};
        for (int c = cl; c < kchunks; c += lpk) {
          float kf[8];
          expand(load_raw(kr + c * 8), kf);
#pragma unroll
          for (int hh = 0; hh < SR_HEADS; ++hh) {
            if (h0 + hh >= HG) break;
            const float4 a = *reinterpret_cast<const float4*>(qs + (h0 + hh) * KL + c * 8);
            const float4 b = *reinterpret_cast<const float4*>(qs + (h0 + hh) * KL + c * 8 + 4);
            float s = dot[hh];
            s = fmaf(a.x, kf[0], s);
            s = fmaf(a.y, kf[1], s);
            s = fmaf(a.z, kf[2], s);
            s = fmaf(a.w, kf[3], s);
            s = fmaf(b.x, kf[4], s);
            s = fmaf(b.y, kf[5], s);
            s = fmaf(b.z, kf[6], s);
            dot[hh] = fmaf(b.w, kf[7], s);
          }
        }
#pragma unroll
        for (int hh = 0; hh < SR_HEADS; ++hh) {
          if (h0 + hh >= HG) break;
          for (int o = lpk >> 1; o; o >>= 1)
            dot[hh] += __shfl_xor_sync(0xFFFFFFFFu, dot[hh], o);
          if (cl == 0 && in) ws[(h0 + hh) * SR_TILE + key] = dot[hh];
        }
      }
    }
    __syncthreads();
    for (int i = tid; i < HG * SR_TILE; i += SR_THREADS) {
      const int hh = i / SR_TILE, key = i % SR_TILE;
      if (key < n) {
        const int h = g * HG + hh;
        const float s = cap_score<FAST>(ws[i] * p.a.scale, p.a.softcap);
        ws[i] = sigmoidf<FAST>(s + bias_at(p.a, h, pos - (k0 + key)));
      }
    }
    __syncthreads();
    for (int h0 = 0; h0 < HG; h0 += SR_HEADS) {
      for (int v0 = vc; v0 < vchunks; v0 += SR_THREADS) {  // one trip unless v_ld > 1024
        float acc[SR_HEADS][8] = {};
        if (kg < kgroups) {
#pragma unroll 4
          for (int key = kg; key < n; key += kgroups) {
            const uint32_t j = k0 + key;
            const E* vr;
            if (owns_new && j == pos) {
              vr = newv;
            } else {
              const uint32_t block = min(table[j / BS], kv.num_blocks - 1);
              vr = pool + kv.v_elem(block, g, j % BS);
            }
            float vf[8];
            expand(load_raw(vr + v0 * 8), vf);
#pragma unroll
            for (int hh = 0; hh < SR_HEADS; ++hh) {
              const float w = h0 + hh < HG ? ws[(h0 + hh) * SR_TILE + key] : 0.f;
#pragma unroll
              for (int e = 0; e < 8; ++e) acc[hh][e] = fmaf(w, vf[e], acc[hh][e]);
            }
          }
#pragma unroll
          for (int hh = 0; hh < SR_HEADS; ++hh)
#pragma unroll
            for (int e = 0; e < 8; ++e)
              redv[((size_t)kg * SR_HEADS + hh) * VL + v0 * 8 + e] = acc[hh][e];
        }
      }
      __syncthreads();
      for (int i = tid; i < SR_HEADS * VL; i += SR_THREADS) {
        const int hh = i / VL;
        if (h0 + hh < HG) {
          float s = 0.f;
          for (int k = 0; k < kgroups; ++k) s += redv[(size_t)k * SR_HEADS * VL + i];
          acc_s[h0 * VL + i] += s;
        }
      }
      __syncthreads();
    }
  }

  auto store = [&](int hh, int d, float v) {
    const int64_t at = t * p.out_ld + (int64_t)(g * HG + hh) * DV + d;
    if (p.out_f32)
      static_cast<float*>(p.out)[at] = v;
    else
      static_cast<E*>(p.out)[at] = to_elem<E>(v);
  };
  if (n_parts == 1) {
    for (int i = tid; i < HG * DV; i += SR_THREADS) {
      const int hh = i / DV, d = i - hh * DV;
      store(hh, d, acc_s[hh * VL + d]);
    }
    return;
  }
  // shares of a row: published, and added in order by the CTA that arrives last
  float* mine = p.partial + ((size_t)t * H + (size_t)g * HG) * p.parts * DV;
  for (int i = tid; i < HG * DV; i += SR_THREADS) {
    const int hh = i / DV, d = i - hh * DV;
    mine[((size_t)hh * p.parts + part) * DV + d] = acc_s[hh * VL + d];
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) ticket = atomicAdd(&p.tickets[t * G + g], 1u);
  __syncthreads();
  if (ticket != n_parts - 1) return;
  __threadfence();
  for (int i = tid; i < HG * DV; i += SR_THREADS) {
    const int hh = i / DV, d = i - hh * DV;
    float s = 0.f;
    for (uint32_t k = 0; k < n_parts; ++k)
      s += __ldcg(&mine[((size_t)hh * p.parts + k) * DV + d]);
    store(hh, d, s);
  }
  if (tid == 0) p.tickets[t * G + g] = 0;
}

// ------------------------------------------------- one query row's heads as a tile (bf16) ----
// The same work as sigmoid_rows_kernel with the group's query heads as the 16 rows of an mma tile
// (blockIdx.y = kv head and block of 16 heads). The four warps take 16-key slices in turn; each
// streams its own through a ring of two in shared memory, so no warp waits for another before
// the end. In the decode step the pool's rows are requested before the wait for the kernel in
// front (a step's first kernel starts only when everything before the step has ended, so the
// rows of earlier steps are there); the step's own row, which is not stored yet, is patched in.
constexpr int SG_THREADS = 128, SG_WARPS = 4, SG_KEYS = 16, SG_RING = 2;

template <int VT>
__global__ void __launch_bounds__(SG_THREADS) sigmoid_group_kernel(const RowsArgs p) {
  extern __shared__ __align__(16) uint8_t sm_raw[];
  __shared__ float red[32];
  __shared__ uint32_t ticket;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const KvDenseLayer& kv = p.kv;
  const int G = kv.kv_heads, H = p.a.heads, HG = H / G, HB = (HG + 15) / 16;
  const int part = blockIdx.x, g = blockIdx.y / HB, h0 = blockIdx.y % HB * 16;
  const int64_t t = blockIdx.z;
  const int nh = min(16, HG - h0);  // heads of this CTA
  const int D = kv.k_dim, DV = kv.v_dim, KL = kv.k_ld, VL = kv.v_ld, BS = kv.block_size;
  const int dp = (D + 15) & ~15, ks = dp + 8;
  constexpr int vs = VT * 8 + 8;
  bf16* Qs = reinterpret_cast<bf16*>(sm_raw);            // [16][ks]
  bf16* newk = Qs + 16 * ks;                             // [dp]
  bf16* newv = newk + dp;                                // [VT * 8]
  bf16* ring0 = newv + VT * 8;
  const int slot_elems = SG_KEYS * (ks + vs);
  bf16* ring = ring0 + (size_t)warp * SG_RING * slot_elems;
  float* sums = reinterpret_cast<float*>(ring0);         // the ring again, after the keys

  pdl_launch_dependents();
  // positions and tables are step inputs, written before the step's first kernel
  const uint32_t pos = p.map.positions[t];
  const uint32_t seq = p.map.row_seq ? p.map.row_seq[t] : (uint32_t)t;
  const uint32_t* table = p.map.tables + (size_t)seq * p.map.max_blocks;
  const uint32_t lo = p.a.window && pos + 1 > p.a.window ? pos + 1 - p.a.window : 0;
  const uint32_t n_units = (pos + 1 - lo + SR_TILE - 1) / SR_TILE;
  const uint32_t per = (n_units + p.parts - 1) / p.parts;
  const uint32_t n_parts = (n_units + per - 1) / per;
  if ((uint32_t)part >= n_parts) return;
  const uint32_t k_begin = lo + part * per * SR_TILE;
  const uint32_t k_end = min(pos + 1, k_begin + per * SR_TILE);
  const bool fused = p.q == nullptr;
  const bool owns_new = fused && k_end == pos + 1;
  const bf16* pool = reinterpret_cast<const bf16*>(kv.base);
  const int slices = (int)((k_end - k_begin + SG_KEYS - 1) / SG_KEYS);
  const int mine = slices > warp ? (slices - warp + SG_WARPS - 1) / SG_WARPS : 0;

  const int kc = dp / 8, kl = KL / 8, vl = VL / 8;
  // Lane r (and r + 16) looks up the page of the slice's key r, one slice ahead of its use. The
  // copies run along the rows, so that a warp's requests are whole lines.
  const uint32_t NONE = 0xFFFFFFFFu;
  constexpr uint32_t STRIDE = SG_WARPS * SG_KEYS;  // keys from one slice of a warp to its next
  const uint32_t j0 = k_begin + (uint32_t)warp * SG_KEYS + (lane & 15);
  const uint32_t place0 = j0 / BS, off0 = j0 % BS;
  const bool even = STRIDE % (uint32_t)BS == 0;  // the place inside the page stays the same
  const uint32_t place_step = STRIDE / (uint32_t)BS;
  auto page_of = [&](int i) {
    const uint32_t j = j0 + (uint32_t)i * STRIDE;
    return i < mine && j < k_end && !(owns_new && j == pos)
               ? table[even ? place0 + (uint32_t)i * place_step : j / BS]
               : NONE;
  };
  const int kr0 = lane / kc, kc0 = lane % kc, kr_step = 32 / kc, kc_step = 32 % kc;
  auto fetch = [&](int i, uint32_t block) {
    if (i < mine) {
      bf16* kd = ring + (size_t)(i % SG_RING) * slot_elems;
      bf16* vd = kd + SG_KEYS * ks;
      const bool in = block < kv.num_blocks;
      if (!in && block != NONE) atomicOr(p.status, DEV_BAD_INDEX);
      const uint32_t off = even ? off0 : (j0 + (uint32_t)i * STRIDE) % BS;
      // row offsets in 16-byte units
      const uint32_t ku = in ? (uint32_t)(kv.k_elem(block, g, off) / 8) : NONE;
      const uint32_t vu = in ? (uint32_t)(kv.v_elem(block, g, off) / 8) : NONE;
      int r = kr0, c = kc0;
      for (int n = 0; n < kc / 2; ++n) {
        const uint32_t u = __shfl_sync(0xFFFFFFFFu, ku, r);
        const bool ok = u != NONE && c < kl;
        cp_async16(kd + r * ks + c * 8, ok ? pool + (size_t)(u + c) * 8 : pool, ok);
        r += kr_step;
        c += kc_step;
        if (c >= kc) {
          c -= kc;
          ++r;
        }
      }
#pragma unroll
      for (int n = 0; n < VT / 2; ++n) {
        const int vr = (lane + 32 * n) / VT, vcol = (lane + 32 * n) % VT;
        const uint32_t u = __shfl_sync(0xFFFFFFFFu, vu, vr);
        const bool ok = u != NONE && vcol < vl;
        cp_async16(vd + vr * vs + vcol * 8, ok ? pool + (size_t)(u + vcol) * 8 : pool, ok);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const uint32_t page0 = page_of(0);
  uint32_t ahead = page_of(1);
  // Decoding: the rows were stored by earlier steps. Otherwise the kernel in front stored some.
  if (fused) fetch(0, page0);
  for (int i = tid; i < 16 * ks / 8; i += SG_THREADS)
    reinterpret_cast<uint4*>(Qs)[i] = make_uint4(0u, 0u, 0u, 0u);
  pdl_wait();
  if (!fused) fetch(0, page0);

  if (!fused) {
    const bf16* q = static_cast<const bf16*>(p.q) + ((size_t)t * H + (size_t)g * HG + h0) * KL;
    __syncthreads();
    for (int i = tid; i < nh * kl; i += SG_THREADS) {
      const int r = i / kl, c = i - r * kl;
      reinterpret_cast<uint4*>(Qs + r * ks)[c] = reinterpret_cast<const uint4*>(q + r * KL)[c];
    }
  } else {
    const int nq = H * D, nk = G * D;
    const float* src = p.s.qkv + t * (int64_t)(nq + nk + G * DV);
    auto value = [&](int i) {
      float v = src[i];
      for (int r = 1; r < p.s.parts; ++r) v += src[r * p.s.part_stride + i];
      return v;
    };
    // four at a time where rows and heads allow it: every trip is one access time
    const bool four = D % 4 == 0 && (G * DV) % 4 == 0 && p.s.part_stride % 4 == 0;
    auto value4 = [&](int i) {
      float4 v = *reinterpret_cast<const float4*>(src + i);
      for (int r = 1; r < p.s.parts; ++r) {
        const float4 u = *reinterpret_cast<const float4*>(src + r * p.s.part_stride + i);
        v.x += u.x, v.y += u.y, v.z += u.z, v.w += u.w;
      }
      return v;
    };
    auto squares = [&](int first, int n) {
      float acc = 0.f;
      if (four) {
#pragma unroll 4
        for (int i = tid * 4; i < n; i += SG_THREADS * 4) {
          const float4 v = value4(first + i);
          acc += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
      } else {
        for (int i = tid; i < n; i += SG_THREADS) {
          const float v = value(first + i);
          acc += v * v;
        }
      }
      return acc;
    };
    float ss = squares(0, nq), sk = owns_new ? squares(nq, nk) : 0.f;
    ss = block_sum(ss, red);
    float inv = 1.0f / sqrtf(ss / (float)nq + p.s.eps);
    const int q0 = (g * HG + h0) * D;  // this CTA's heads lie one after the other
    if (four) {
      for (int i = tid * 4; i < nh * D; i += SG_THREADS * 4) {
        const int r = i / D, d = i - r * D;
        const float4 v = value4(q0 + i);
        const float* w = p.s.q_norm + q0 + i;
        uint2 pk = make_uint2(pack_bf16(v.x * inv * w[0], v.y * inv * w[1]),
                              pack_bf16(v.z * inv * w[2], v.w * inv * w[3]));
        *reinterpret_cast<uint2*>(Qs + r * ks + d) = pk;
      }
    } else {
      for (int i = tid; i < nh * D; i += SG_THREADS) {
        const int r = i / D, d = i - r * D;
        Qs[r * ks + d] = to_elem<bf16>(value(q0 + i) * inv * p.s.q_norm[q0 + i]);
      }
    }
    if (owns_new) {
      sk = block_sum(sk, red);
      inv = 1.0f / sqrtf(sk / (float)nk + p.s.eps);
      const uint32_t place = pos / BS;
      uint32_t block = kv.num_blocks;
      if (place < p.map.max_blocks) block = table[place];
      const bool ok = block < kv.num_blocks;
      if (!ok && tid == 0) atomicOr(p.status, DEV_BAD_INDEX);
      const bool store = ok && h0 == 0;  // one of the group's CTAs
      bf16* wp = reinterpret_cast<bf16*>(kv.base);
      for (int d = tid; d < dp; d += SG_THREADS) {
        const bf16 v =
            to_elem<bf16>(d < D ? value(nq + g * D + d) * inv * p.s.k_norm[g * D + d] : 0.f);
        newk[d] = v;
        if (store && d < KL) wp[kv.k_elem(block, g, pos % BS) + d] = v;
      }
      for (int d = tid; d < VT * 8; d += SG_THREADS) {
        const bf16 v = to_elem<bf16>(d < DV ? value(nq + nk + g * DV + d) : 0.f);
        newv[d] = v;
        if (store && d < VL) wp[kv.v_elem(block, g, pos % BS) + d] = v;
      }
    }
  }
  __syncthreads();

  float o[VT][4];
#pragma unroll
  for (int i = 0; i < VT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int nvt = (DV + 7) / 8, row = lane >> 2;
  const float cap = p.a.softcap;
  // the distance term is computed: its table would be read from the second-level cache
  const int head0 = g * HG + h0 + min(row, nh - 1), head1 = g * HG + h0 + min(row + 8, nh - 1);
  const float LN2 = 0.69314718055994530942f;
  const float far0 = p.a.r1[head0] * LN2, far1 = p.a.r1[head1] * LN2;
  const float rate0 = p.a.r2[head0], rate1 = p.a.r2[head1];
  const float pb0 = p.a.pb[head0], pb1 = p.a.pb[head1];
  const uint32_t qa = smem_u32(Qs) + (uint32_t)((lane & 15) * ks + (lane >> 4) * 8) * 2;
  for (int i = 0; i < mine; ++i) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncwarp();
    fetch(i + 1, ahead);  // into the slot that the step before this one has left
    ahead = page_of(i + 2);
    bf16* kd = ring + (size_t)(i % SG_RING) * slot_elems;
    bf16* vd = kd + SG_KEYS * ks;
    const uint32_t k0 = k_begin + (uint32_t)(warp + i * SG_WARPS) * SG_KEYS;
    if (owns_new && pos - k0 < SG_KEYS) {
      for (int d = lane; d < dp; d += 32) kd[(pos - k0) * ks + d] = newk[d];
      for (int d = lane; d < VT * 8; d += 32) vd[(pos - k0) * vs + d] = newv[d];
      __syncwarp();
    }
    float s[2][4] = {};
    const uint32_t ka = smem_u32(kd) +
                        (uint32_t)(((lane & 7) + ((lane >> 4) << 3)) * ks + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll 4
    for (int kk = 0; kk < dp; kk += 16) {
      uint32_t a[4], b[4];
      ldm_x4(a, qa + kk * 2);
      ldm_x4(b, ka + kk * 2);
      mma_bf16(s[0], a, b[0], b[1]);
      mma_bf16(s[1], a, b[2], b[3]);
    }
    const float dist = (float)(int)(pos - (k0 + (lane & 3) * 2));
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const uint32_t j = k0 + nt * 8 + (lane & 3) * 2 + (e & 1);
        float w = 0.f;
        if (row + (e >> 1) * 8 < nh && j < k_end) {
          const float d = dist - (float)(nt * 8 + (e & 1));
          const float lg = __log2f(fmaf(e >> 1 ? rate1 : rate0, d, 1.f));
          w = sigmoidf<true>(cap_score<true>(s[nt][e] * p.a.scale, cap) +
                             fmaf(e >> 1 ? -far1 : -far0, lg, e >> 1 ? pb1 : pb0));
        }
        s[nt][e] = w;
      }
    const uint32_t a[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]),
                           pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
    const uint32_t va = smem_u32(vd) + (uint32_t)((lane & 15) * vs + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int nt = 0; nt < VT; nt += 2) {
      if (nt < nvt) {
        uint32_t b[4];
        ldm_x4_t(b, va + nt * 16);
        mma_bf16(o[nt], a, b[0], b[1]);
        mma_bf16(o[nt + 1], a, b[2], b[3]);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();  // the rings are read out
  for (int nt = 0; nt < VT; ++nt) {
    const int c = nt * 8 + (lane & 3) * 2;
    float* r0 = sums + ((size_t)warp * 16 + row) * (VT * 8) + c;
    r0[0] = o[nt][0], r0[1] = o[nt][1];
    float* r1 = r0 + (size_t)8 * VT * 8;
    r1[0] = o[nt][2], r1[1] = o[nt][3];
  }
  __syncthreads();
  auto total = [&](int hh, int d) {
    float v = 0.f;
    for (int w = 0; w < SG_WARPS; ++w) v += sums[((size_t)w * 16 + hh) * (VT * 8) + d];
    return v;
  };
  auto store = [&](int hh, int d, float v) {
    const int64_t at = t * p.out_ld + (int64_t)(g * HG + h0 + hh) * DV + d;
    if (p.out_f32)
      static_cast<float*>(p.out)[at] = v;
    else
      static_cast<bf16*>(p.out)[at] = to_elem<bf16>(v);
  };
  float* mine_p = p.partial + ((size_t)t * H + (size_t)g * HG + h0) * p.parts * DV;
  for (int i = tid; i < nh * DV; i += SG_THREADS) {
    const int hh = i / DV, d = i - hh * DV;
    if (n_parts == 1)
      store(hh, d, total(hh, d));
    else
      mine_p[((size_t)hh * p.parts + part) * DV + d] = total(hh, d);
  }
  if (n_parts == 1) return;
  __threadfence();
  __syncthreads();
  uint32_t* tk = &p.tickets[(t * G + g) * HB + blockIdx.y % HB];
  if (tid == 0) ticket = atomicAdd(tk, 1u);
  __syncthreads();
  if (ticket != n_parts - 1) return;
  __threadfence();
  if (DV % 4 == 0) {
    for (int i = tid * 4; i < nh * DV; i += SG_THREADS * 4) {
      const int hh = i / DV, d = i - hh * DV;
      const float* src = mine_p + (size_t)hh * p.parts * DV + d;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
      for (uint32_t k = 0; k < n_parts; ++k) {
        const float4 u = __ldcg(reinterpret_cast<const float4*>(src + (size_t)k * DV));
        v.x += u.x, v.y += u.y, v.z += u.z, v.w += u.w;
      }
      store(hh, d, v.x), store(hh, d + 1, v.y), store(hh, d + 2, v.z), store(hh, d + 3, v.w);
    }
  } else {
    for (int i = tid; i < nh * DV; i += SG_THREADS) {
      const int hh = i / DV, d = i - hh * DV;
      float v = 0.f;
      for (uint32_t k = 0; k < n_parts; ++k)
        v += __ldcg(&mine_p[((size_t)hh * p.parts + k) * DV + d]);
      store(hh, d, v);
    }
  }
  if (tid == 0) *tk = 0;
}

// ------------------------------------------------------------------ 64-row tiles (bf16) ----
constexpr int ST_THREADS = 128;
constexpr int ST_Q = 64, ST_K = 64;
constexpr uint32_t ST_BIAS_SMEM = 4096;  // table entries that are staged in shared memory

struct TilesArgs {
  SigmoidAttn a;
  KvDenseLayer kv;
  RowMap map;
  const bf16* q;
  const AttnTile* tiles;
  void* out;
  int64_t out_ld;
  int out_f32;
  int dp;          // k_dim rounded up to 16
  int bias_n;      // staged table entries per head
  int* status;
};

// VT = value columns / 8, rounded up to an even template size
template <int VT>
__global__ void __launch_bounds__(ST_THREADS) sigmoid_tiles_kernel(const TilesArgs p) {
  extern __shared__ __align__(16) uint8_t sm_raw[];
  __shared__ int64_t koff[2][ST_K];  // element offset of a key's row in the pool, -1: none
  __shared__ int64_t voff[2][ST_K];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const KvDenseLayer& kv = p.kv;
  const int H = p.a.heads, HG = H / (int)kv.kv_heads, h = blockIdx.y, g = h / HG;
  const int DV = kv.v_dim, KL = kv.k_ld, VL = kv.v_ld, BS = kv.block_size;
  const int ks = p.dp + 8;          // row stride of Q and K, elements
  constexpr int vs = VT * 8 + 8;    // row stride of V
  bf16* Qs = reinterpret_cast<bf16*>(sm_raw);
  bf16* Ks = Qs + ST_Q * ks;        // two buffers
  bf16* Vs = Ks + 2 * ST_K * ks;
  float* tab = reinterpret_cast<float*>(Vs + 2 * ST_K * vs);  // -log2(e) * (cap + bias)

  pdl_launch_dependents();
  const AttnTile tile = p.tiles[blockIdx.x];
  const uint32_t* table = p.map.tables + (size_t)tile.seq * p.map.max_blocks;
  const uint32_t q_end = tile.pos0 + tile.rows;  // exclusive
  const uint32_t lo =
      p.a.window && tile.pos0 + 1 > p.a.window ? tile.pos0 + 1 - p.a.window : 0;
  const float cap = p.a.softcap;
  const float L2E = 1.44269504088896340736f;
  for (int i = tid; i < p.bias_n; i += ST_THREADS)
    tab[i] = -L2E * (cap + p.a.bias[(size_t)h * p.a.bias_len + i]);
  pdl_wait();

  auto place_keys = [&](uint32_t k0, int buf) {
    if (tid < ST_K) {
      const uint32_t j = k0 + tid;
      int64_t ko = -1, vo = -1;
      if (j < q_end) {
        const uint32_t block = table[j / BS];
        if (block < kv.num_blocks) {
          ko = (int64_t)kv.k_elem(block, g, j % BS);
          vo = (int64_t)kv.v_elem(block, g, j % BS);
        } else {
          atomicOr(p.status, DEV_BAD_INDEX);
        }
      }
      koff[buf][tid] = ko;
      voff[buf][tid] = vo;
    }
  };
  const bf16* pool = reinterpret_cast<const bf16*>(kv.base);
  auto load_keys = [&](int buf) {
    const int kc = p.dp / 8, kl = KL / 8, vl = VL / 8;
    for (int i = tid; i < ST_K * kc; i += ST_THREADS) {
      const int r = i / kc, c = i - r * kc;
      const int64_t o = koff[buf][r];
      const bool in = o >= 0 && c < kl;
      cp_async16(Ks + (size_t)(buf * ST_K + r) * ks + c * 8, in ? pool + o + c * 8 : pool, in);
    }
    for (int i = tid; i < ST_K * VT; i += ST_THREADS) {
      const int r = i / VT, c = i - r * VT;
      const int64_t o = voff[buf][r];
      const bool in = o >= 0 && c < vl;
      cp_async16(Vs + (size_t)(buf * ST_K + r) * vs + c * 8, in ? pool + o + c * 8 : pool, in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  {
    const int kc = p.dp / 8, kl = KL / 8;
    for (int i = tid; i < ST_Q * kc; i += ST_THREADS) {
      const int r = i / kc, c = i - r * kc;
      const bool in = (uint32_t)r < tile.rows && c < kl;
      const bf16* src = p.q + ((size_t)(tile.row0 + (in ? r : 0)) * H + h) * KL + (in ? c : 0) * 8;
      cp_async16(Qs + (size_t)r * ks + c * 8, src, in);
    }
  }
  place_keys(lo, 0);
  __syncthreads();
  load_keys(0);

  float o[VT][4];
#pragma unroll
  for (int i = 0; i < VT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int row_in = warp * 16 + (lane >> 2);           // first of the lane's two rows
  const int qpos0 = (int)tile.pos0 + row_in;
  const float k1 = cap != 0.f ? p.a.scale * 2.f * L2E / cap : 0.f;
  const float c1 = 2.f * cap * L2E;
  const int window = p.a.window ? (int)min(p.a.window, 0x7FFFFFFFu) : 0x7FFFFFFF;
  const int nvt = (DV + 7) / 8;

  int buf = 0;
  for (uint32_t k0 = lo; k0 < q_end; k0 += ST_K, buf ^= 1) {
    if (k0 + ST_K < q_end) place_keys(k0 + ST_K, buf ^ 1);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this tile has landed, the other buffer is free and its places are known
    if (k0 + ST_K < q_end) load_keys(buf ^ 1);

    // a warp's rows may lie wholly before this tile's keys or past the window
    const int w_first = (int)tile.pos0 + warp * 16, w_last = w_first + 15;
    if ((int)k0 > w_last || w_first - (int)(k0 + ST_K - 1) >= window) continue;

    float s[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    const uint32_t qa = smem_u32(Qs) + (uint32_t)(((warp * 16 + (lane & 15)) * ks + (lane >> 4) * 8) * 2);
    const uint32_t ka = smem_u32(Ks) +
                        (uint32_t)(((buf * ST_K + (lane & 7) + ((lane >> 4) << 3)) * ks +
                                    ((lane >> 3) & 1) * 8) * 2);
#pragma unroll 2
    for (int kk = 0; kk < p.dp; kk += 16) {
      uint32_t a[4];
      ldm_x4(a, qa + kk * 2);
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        uint32_t b[4];
        ldm_x4(b, ka + (uint32_t)(nt * 16 * ks + kk) * 2);
        mma_bf16(s[2 * nt], a, b[0], b[1]);
        mma_bf16(s[2 * nt + 1], a, b[2], b[3]);
      }
    }
    // weights
    const bool whole = w_first - (int)(k0 + ST_K - 1) >= 0 && w_last - (int)k0 < window;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = qpos0 + (e >> 1) * 8 - (int)(k0 + nt * 8 + (lane & 3) * 2 + (e & 1));
        float b;
        if (p.bias_n) {
          b = tab[min(max(d, 0), p.bias_n - 1)];
        } else {
          b = -L2E * (cap + bias_at(p.a, h, (uint32_t)max(d, 0)));
        }
        float arg;  // -log2(e) * (score + bias)
        if (cap != 0.f)
          arg = fmaf(rcp_approx(1.f + ex2_approx(s[nt][e] * k1)), c1, b);
        else
          arg = fmaf(s[nt][e], -L2E * p.a.scale, b);
        float w = rcp_approx(1.f + ex2_approx(arg));
        if (!whole && (d < 0 || d >= window)) w = 0.f;
        s[nt][e] = w;
      }
    const uint32_t va = smem_u32(Vs) +
                        (uint32_t)(((buf * ST_K + (lane & 15)) * vs + (lane >> 4) * 8) * 2);
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      const uint32_t a[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]),
                             pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                             pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]),
                             pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
      for (int nt = 0; nt < VT; nt += 2) {
        if (nt < nvt) {
          uint32_t b[4];
          ldm_x4_t(b, va + (uint32_t)(kk * 16 * vs + nt * 8) * 2);
          mma_bf16(o[nt], a, b[0], b[1]);
          mma_bf16(o[nt + 1], a, b[2], b[3]);
        }
      }
    }
  }
#pragma unroll
  for (int nt = 0; nt < VT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = row_in + (e >> 1) * 8, c = nt * 8 + (lane & 3) * 2 + (e & 1);
      if ((uint32_t)r < tile.rows && c < DV) {
        const int64_t at = (int64_t)(tile.row0 + r) * p.out_ld + (int64_t)h * DV + c;
        if (p.out_f32)
          static_cast<float*>(p.out)[at] = o[nt][e];
        else
          static_cast<bf16*>(p.out)[at] = to_elem<bf16>(o[nt][e]);
      }
    }
}

int32_t make_sigmoid_attn(kanso_cuda_ctx* ctx, uint32_t heads, uint32_t window, float scale,
                          float softcap, const float* r1, const float* r2, const float* pb,
                          SigmoidAttn* out, void** mem) {
  const uint32_t len = window ? std::min(window, ATTN_BIAS_MAX) : ATTN_BIAS_MAX;
  std::vector<float> host(3 * (size_t)heads + (size_t)heads * len, 0.f);
  float *a = host.data(), *b = a + heads, *c = b + heads, *tab = c + heads;
  for (uint32_t h = 0; h < heads; ++h) {
    a[h] = r1 ? r1[h] : 0.f;
    b[h] = r2 ? r2[h] : 0.f;
    c[h] = pb ? pb[h] : 0.f;
    for (uint32_t d = 0; d < len; ++d)
      tab[(size_t)h * len + d] =
          (float)((double)c[h] - (double)a[h] * std::log1p((double)b[h] * (double)d));
  }
  float* dev = nullptr;
  KANSO_CUDA_TRY(ctx, cudaMalloc((void**)&dev, host.size() * 4), "attention constants");
  *mem = dev;
  KANSO_CUDA_TRY(ctx, cudaMemcpy(dev, host.data(), host.size() * 4, cudaMemcpyHostToDevice),
                 "attention constants");
  *out = SigmoidAttn();
  out->heads = heads;
  out->window = window;
  out->scale = scale;
  out->softcap = softcap;
  out->r1 = dev;
  out->r2 = dev + heads;
  out->pb = dev + 2 * heads;
  out->bias = dev + 3 * heads;
  out->bias_len = len;
  return KANSO_OK;
}

template <int VT>
static int32_t group_launch(kanso_cuda_ctx* ctx, dim3 grid, size_t smem, const RowsArgs& p) {
  int32_t st = allow_max_smem(ctx, (const void*)sigmoid_group_kernel<VT>);
  if (st) return st;
  const cudaError_t e =
      launch_dependent(ctx, sigmoid_group_kernel<VT>, grid, dim3(SG_THREADS), smem, p);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "sigmoid attention launch");
  return after_launch(ctx, "sigmoid_group");
}

int32_t launch_sigmoid_attn_rows(kanso_cuda_ctx* ctx, int32_t compute, const SigmoidAttn& a,
                                 const KvDenseLayer& kv, const void* q, const QkvSource* fused,
                                 const RowMap& map, uint32_t max_keys, void* out, bool out_f32,
                                 int64_t out_ld, int64_t T) {
  if (T > 65535)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "attention: %lld rows in one launch", (long long)T);
  const uint32_t G = kv.kv_heads, HG = a.heads / G, HB = (HG + 15) / 16;
  RowsArgs p;
  p.a = a;
  p.kv = kv;
  p.map = map;
  p.q = fused ? nullptr : q;
  if (fused) p.s = *fused;
  p.out = out;
  p.out_ld = out_ld;
  p.out_f32 = out_f32;
  p.status = ctx->dev_status;
  p.tickets = ctx->pa_tickets;
  p.partial = nullptr;
  // bfloat16 with the sizes of the mma form
  const int dp = (int)((kv.k_dim + 15u) & ~15u);
  const int vt = kv.v_dim <= 32 ? 4 : kv.v_dim <= 64 ? 8 : kv.v_dim <= 128 ? 16 : 32;
  const size_t gsmem =
      ((size_t)16 * (dp + 8) + dp + vt * 8 +
       std::max<size_t>((size_t)SG_WARPS * SG_RING * SG_KEYS * (dp + 8 + vt * 8 + 8),
                        (size_t)SG_WARPS * 16 * vt * 8 * 2)) * 2;
  // (a pool's rows must be countable in 32 bits of 16-byte units)
  const bool group = compute == KANSO_COMPUTE_BF16 && kv.v_dim <= 256 && kv.k_dim <= 512 &&
                     gsmem <= 220 * 1024 &&
                     (uint64_t)kv.num_blocks * kv.kv_heads * kv.rec_elems / 8 < 0xFFFFFFFFull;
  if (a.window) max_keys = std::min(max_keys, a.window);
  const uint32_t tiles = std::max(1u, (max_keys + SR_TILE - 1) / SR_TILE);
  // Shares of the keys. The mma form: the split with the shortest run of waves, a wave being a
  // share's tiles and about three tiles' worth of fixed work; the plain form: four CTAs per SM.
  const uint64_t ctas = (uint64_t)T * G * (group ? HB : 1);
  uint32_t parts = 1;
  if (ctas <= kanso_cuda_ctx::kPaTickets) {
    if (group) {
      const uint64_t per_sm = std::max<uint64_t>(
          1, std::min<uint64_t>(4, (uint64_t)ctx->smem_per_sm / (gsmem + 1200)));
      const uint64_t resident = (uint64_t)ctx->sm_count * per_sm;
      uint64_t best = ~0ull;
      for (uint32_t n = 1; n <= tiles; ++n) {
        const uint64_t cost = (ctas * n + resident - 1) / resident * ((tiles + n - 1) / n + 3);
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
  parts = (tiles + per - 1) / per;
  p.parts = parts;
  if (parts > 1) {
    p.partial = (float*)ctx_scratch(ctx, (size_t)T * a.heads * parts * kv.v_dim * 4);
    if (!p.partial) return KANSO_ERR_DEVICE;
  }
  if (group) {
    const dim3 grid(parts, G * HB, (unsigned)T);
    switch (vt) {
      case 4: return group_launch<4>(ctx, grid, gsmem, p);
      case 8: return group_launch<8>(ctx, grid, gsmem, p);
      case 16: return group_launch<16>(ctx, grid, gsmem, p);
      default: return group_launch<32>(ctx, grid, gsmem, p);
    }
  }
  const int vchunks = kv.v_ld / 8, kgroups = std::max(1, std::min(SR_THREADS / vchunks, 16));
  const size_t smem = ((size_t)HG * kv.k_ld + (size_t)HG * SR_TILE + (size_t)HG * kv.v_ld +
                       (size_t)kgroups * SR_HEADS * kv.v_ld) * 4 +
                      ((size_t)kv.k_ld + kv.v_ld) * (compute == KANSO_COMPUTE_BF16 ? 2 : 4);
  if (smem > 220 * 1024)
    return fail(ctx, KANSO_ERR_UNSUPPORTED,
                "attention: %u query heads per key/value head of %u and %u columns", HG, kv.k_dim,
                kv.v_dim);
  auto kern = compute == KANSO_COMPUTE_BF16 ? sigmoid_rows_kernel<bf16> : sigmoid_rows_kernel<float>;
  int32_t st = allow_max_smem(ctx, (const void*)kern);
  if (st) return st;
  const cudaError_t e = launch_dependent(ctx, kern, dim3(parts, G, (unsigned)T), dim3(SR_THREADS),
                                         smem, p);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "sigmoid attention launch");
  return after_launch(ctx, "sigmoid_rows");
}

template <int VT>
static int32_t tiles_launch(kanso_cuda_ctx* ctx, dim3 grid, size_t smem, const TilesArgs& p) {
  int32_t st = allow_max_smem(ctx, (const void*)sigmoid_tiles_kernel<VT>);
  if (st) return st;
  const cudaError_t e =
      launch_dependent(ctx, sigmoid_tiles_kernel<VT>, grid, dim3(ST_THREADS), smem, p);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "sigmoid attention launch");
  return after_launch(ctx, "sigmoid_tiles");
}

int32_t launch_sigmoid_attn_tiles(kanso_cuda_ctx* ctx, const SigmoidAttn& a,
                                  const KvDenseLayer& kv, const void* q, const RowMap& map,
                                  const AttnTile* tiles, uint32_t n_tiles, void* out,
                                  bool out_f32, int64_t out_ld, bool* handled) {
  *handled = false;
  if (kv.k_dim > 256 || kv.v_dim > 256 || a.heads > 65535) return KANSO_OK;
  TilesArgs p;
  p.a = a;
  p.kv = kv;
  p.map = map;
  p.q = static_cast<const bf16*>(q);
  p.tiles = tiles;
  p.out = out;
  p.out_ld = out_ld;
  p.out_f32 = out_f32;
  p.status = ctx->dev_status;
  p.dp = (int)((kv.k_dim + 15u) & ~15u);
  // the whole table of a head in shared memory when every visible distance lies in it
  p.bias_n = a.window && a.window <= std::min(a.bias_len, ST_BIAS_SMEM) ? (int)a.window : 0;
  const int vt = kv.v_dim <= 32 ? 4 : kv.v_dim <= 64 ? 8 : kv.v_dim <= 128 ? 16 : 32;
  const size_t smem = (size_t)(ST_Q + 2 * ST_K) * (p.dp + 8) * 2 +
                      (size_t)2 * ST_K * (vt * 8 + 8) * 2 + (size_t)p.bias_n * 4;
  if (smem > 220 * 1024) return KANSO_OK;
  *handled = true;
  const dim3 grid(n_tiles, a.heads);
  switch (vt) {
    case 4: return tiles_launch<4>(ctx, grid, smem, p);
    case 8: return tiles_launch<8>(ctx, grid, smem, p);
    case 16: return tiles_launch<16>(ctx, grid, smem, p);
    default: return tiles_launch<32>(ctx, grid, smem, p);
  }
}

}  // namespace kanso
