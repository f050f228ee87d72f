// Causal softmax attention of prompts on tcgen05 (bfloat16): 128 query rows of one head against key
// tiles of 64, keys and values one after the other in memory. Keys and queries may have a second
// part (rotated columns) of which the keys' is shared by all heads; the softmax's denominator may
// hold one more term per head that has no key and no value (a sink).
//
//   warps 8, 10  copies by tensor map, panels of 64 columns (128-byte swizzle): the query tile once
//              and a ring of key tiles; a ring of value tiles. Two warps, since a value tile's place
//              is free much later than a key tile's, which would wait behind it.
//   warp 9     issues S = Q K^T (M = 128, N = 64) into one of two score buffers
//   warp 11    issues O += P V (V N-major) into one of two output accumulators. A thread of its own:
//              in turns with the scores' it would spend a tile's time on waits and issues alone.
//   warps 0-7  two groups of four, each with a score buffer, a weight buffer and an output
//              accumulator of its own: group g takes every second tile. A thread owns a query row.
//
// Each group keeps a reference maximum per row. It only moves, and the group's accumulator is only
// rescaled, when a row's maximum rises by more than 2^8 above it; weights up to 2^8 lose nothing in
// bfloat16. The two groups' results meet at the end.
#include <algorithm>

#include "dense.cuh"
#include "tc05.cuh"
#include "tensor_map.h"
#include "warp_mma.cuh"

namespace kanso {

constexpr int SX_Q = 128, SX_K = 64, SX_MAX_STAGES = 4;
constexpr int SX_WORKERS = 256, SX_THREADS = 384;
constexpr int SX_P_BYTES = SX_Q * SX_K * 2;
constexpr float SX_SLACK = 8.f;

struct SoftmaxArgs {
  const AttnTile* tiles;
  const float* sink;
  bf16* out;
  int64_t out_ld;
  float k1;                // scale * log2(e)
  int v_dim, nv, o_step;   // nv: v_dim rounded up to 16; o_step: to 32, between the accumulators
  int k_panels, r_panels, v_panels;  // 64-column panels of K, of its second part and of V
  int k_steps, r_steps;    // 16-column steps of the scores
  int k_stages, v_stages;
  uint32_t tmem_cols;
  int* status;
};

__global__ void __launch_bounds__(SX_THREADS, 1)
    softmax_prefill_kernel(const __grid_constant__ CUtensorMap qmap,
                           const __grid_constant__ CUtensorMap qrmap,
                           const __grid_constant__ CUtensorMap kmap,
                           const __grid_constant__ CUtensorMap krmap,
                           const __grid_constant__ CUtensorMap vmap, const SoftmaxArgs p) {
  extern __shared__ uint8_t raw[];
  __shared__ uint64_t q_full, k_full[SX_MAX_STAGES], k_empty[SX_MAX_STAGES],
      v_full[SX_MAX_STAGES], v_empty[SX_MAX_STAGES], s_full[2], s_free[2], p_full[2], p_free[2], o_full;
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  __shared__ float2 ml[2][SX_Q];  // per group and row: reference maximum, denominator
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.x;
  const int panels = p.k_panels + p.r_panels;
  const uint32_t k_bytes = (uint32_t)panels * SX_K * 128u;
  const uint32_t v_bytes = (uint32_t)p.v_panels * SX_K * 128u;
  const uint32_t q_panel = SX_Q * 128u;
  uint8_t* Qs = raw + ((1024u - (smem_u32(raw) & 1023u)) & 1023u);
  uint8_t* Ks = Qs + (size_t)panels * q_panel;
  uint8_t* Vs = Ks + (size_t)p.k_stages * k_bytes;
  uint8_t* Ps = Vs + (size_t)p.v_stages * v_bytes;

  pdl_launch_dependents();
  if (tid == 0) {
    mbar_init(&q_full, 1);
    mbar_init(&o_full, 1);
    for (int i = 0; i < SX_MAX_STAGES; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_free[i], SX_WORKERS / 64);
      mbar_init(&p_full[i], SX_WORKERS / 64);
      mbar_init(&p_free[i], 1);
    }
    mbar_fence_init();
    abort_flag = 0;
  }
  // the longest rows of all heads first: what is left at the end is short
  const AttnTile tile = p.tiles[gridDim.y - 1 - blockIdx.y];
  const int key0 = (int)tile.seq;
  const int q_end = (int)(tile.pos0 + tile.rows);  // exclusive
  const int n_tiles = (q_end + SX_K - 1) / SX_K;
  // TMEM only once the kernels in front have ended: they may hold or still want some of it
  pdl_wait();
  if (warp == 9) tmem_alloc(&tmem_slot, p.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot, o_tmem = tmem + 2 * SX_K;

  if (warp == 8 || warp == 10) {
    // ---- copies ----
    if (lane == 0) {
      const bool keys = warp == 8;
      const int stages = keys ? p.k_stages : p.v_stages;
      const uint32_t bytes = keys ? k_bytes : v_bytes;
      uint64_t *full = keys ? k_full : v_full, *empty = keys ? k_empty : v_empty;
      if (keys) {
        mbar_arrive_expect_tx(&q_full, (uint32_t)panels * q_panel);
        for (int c = 0; c < panels; ++c) {
          const bool second = c >= p.k_panels;
          tma_load_3d(Qs + (size_t)c * q_panel, second ? &qrmap : &qmap,
                      (second ? c - p.k_panels : c) * 64, h, (int)tile.row0, &q_full);
        }
      }
      int issued = 0;
      for (int i = 0; i < n_tiles; ++i) {
        const int s = i % stages;
        if (!mbar_wait_abort(&empty[s], ((uint32_t)(i / stages) & 1u) ^ 1u, &abort_flag)) break;
        mbar_arrive_expect_tx(&full[s], bytes);
        uint8_t* dst = (keys ? Ks : Vs) + (size_t)s * bytes;
        const int row = key0 + i * SX_K;
        for (int c = 0; c < (keys ? p.k_panels : p.v_panels); ++c)
          tma_load_3d(dst + (size_t)c * SX_K * 128, keys ? &kmap : &vmap, c * 64, h, row, &full[s]);
        for (int c = 0; keys && c < p.r_panels; ++c)
          tma_load_2d(dst + (size_t)(p.k_panels + c) * SX_K * 128, &krmap, c * 64, row, &full[s]);
        issued = i + 1;
      }
      // leave only when every copy has landed (bounded)
      if (keys) mbar_wait_bounded(&q_full, 0);
      for (int i = max(0, issued - stages); i < issued; ++i)
        mbar_wait_bounded(&full[i % stages], (uint32_t)(i / stages) & 1u);
    }
    __syncwarp();
  } else if (warp == 9) {
    // ---- scores ----
    if (lane == 0) {
      const uint32_t idesc = tc_idesc_bf16(SX_Q, SX_K);
      const uint32_t queries = smem_u32(Qs), keys = smem_u32(Ks);
      bool ok = mbar_wait_abort(&q_full, 0, &abort_flag);
      for (int i = 0; i < n_tiles && ok; ++i) {
        const int b = i & 1, s = i % p.k_stages;
        // the group has read the scores of the tile before
        if (i >= 2) ok = mbar_wait_abort(&s_free[b], ((uint32_t)(i >> 1) & 1u) ^ 1u, &abort_flag);
        if (ok) ok = mbar_wait_abort(&k_full[s], (uint32_t)(i / p.k_stages) & 1u, &abort_flag);
        if (!ok) break;
        tc_fence_after();
        const uint32_t k0 = keys + (uint32_t)s * k_bytes, acc = tmem + (uint32_t)b * SX_K;
        tc_mma_panels(acc, queries, k0, q_panel, SX_K * 128u, p.k_steps, idesc, 0);
        tc_mma_panels(acc, queries + (uint32_t)p.k_panels * q_panel,
                      k0 + (uint32_t)p.k_panels * (SX_K * 128u), q_panel, SX_K * 128u, p.r_steps,
                      idesc, 1);
        tc_commit(&s_full[b]);
        tc_commit(&k_empty[s]);
      }
      if (!ok) abort_flag = 1;
    }
    __syncwarp();
  } else if (warp == 11) {
    // ---- weights x values ----
    if (lane == 0) {
      const uint32_t idesc = tc_idesc_bf16(SX_Q, p.nv) | (1u << 16);  // B is N-major
      const uint64_t weights = tc_smem_desc_sw128(smem_u32(Ps));
      const uint64_t values = tc_smem_desc_nmajor(smem_u32(Vs), SX_K * 128u);
      bool ok = true;
      for (int i = 0; i < n_tiles && ok; ++i) {
        const int b = i & 1, s = i % p.v_stages;
        ok = mbar_wait_abort(&v_full[s], (uint32_t)(i / p.v_stages) & 1u, &abort_flag);
        if (ok) ok = mbar_wait_abort(&p_full[b], (uint32_t)(i >> 1) & 1u, &abort_flag);
        if (!ok) break;
        tc_fence_after();
        const uint64_t ad = weights + (uint32_t)b * (SX_P_BYTES >> 4);
        const uint64_t bd = values + (uint32_t)s * (v_bytes >> 4);
        const uint32_t acc = o_tmem + (uint32_t)(b * p.o_step);
        tc_mma_f16(acc, ad, bd, idesc, i > 1);
#pragma unroll
        for (int k = 1; k < SX_K / 16; ++k) tc_mma_f16(acc, ad + 2 * k, bd + 128 * k, idesc, 1);
        tc_commit(&p_free[b]);
        tc_commit(&v_empty[s]);
      }
      if (ok)
        tc_commit(&o_full);
      else
        abort_flag = 1;
    }
    __syncwarp();
  } else {
    // ---- weights ----
    const int wg = warp >> 2, row = (warp & 3) * 32 + lane;
    const uint32_t quarter = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t s_lane = tmem + quarter + (uint32_t)wg * SX_K;
    const uint32_t o_lane = o_tmem + quarter + (uint32_t)(wg * p.o_step);
    uint8_t* prow = Ps + (size_t)wg * SX_P_BYTES + (size_t)row * 128;
    const int pos = (int)tile.pos0 + row;
    float ref = -INFINITY, l = 0.f;
    for (int i = wg; i < n_tiles; i += 2) {
      const uint32_t par = (uint32_t)(i >> 1) & 1u;
      // a warp gives up as one: what follows is done by all its lanes together
      if (!__all_sync(0xFFFFFFFFu, mbar_wait_abort(&s_full[wg], par, &abort_flag))) break;
      tc_fence_after();
      uint32_t r[2][32];
      tmem_ld32(s_lane, r[0]);
      tmem_ld32(s_lane + 32, r[1]);
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_free[wg]);
      if (i * SX_K + SX_K - 1 > (int)tile.pos0) {  // some row does not see all of the tile
        const int seen = pos - i * SX_K;
#pragma unroll
        for (int k = 0; k < 64; ++k)
          if (k > seen) r[k >> 5][k & 31] = __float_as_uint(-INFINITY);
      }
      float top = -INFINITY;
#pragma unroll
      for (int k = 0; k < 64; ++k) top = fmaxf(top, __uint_as_float(r[k >> 5][k & 31]));
      top *= p.k1;  // the scale is positive
      // PV of this group's tile before has ended: its accumulator and weight buffer are free
      if (!__all_sync(0xFFFFFFFFu, mbar_wait_abort(&p_free[wg], par ^ 1u, &abort_flag))) break;
      const bool raise = top > ref + SX_SLACK;
      if (__any_sync(0xFFFFFFFFu, raise)) {
        const float next = raise ? top : ref;
        const float c = raise ? ex2_approx(ref - next) : 1.f;  // ref -inf: 0
        if (i >= 2) {
          tc_fence_after();
          for (int k = 0; k < p.nv; k += 16) {
            uint32_t o[16];
            tmem_ld16(o_lane + k, o);
#pragma unroll
            for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * c);
            tmem_st16(o_lane + k, o);
          }
        }
        l *= c;
        ref = next;
      }
      const float base = ref == -INFINITY ? 0.f : -ref;  // a row that has seen no key yet
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        uint32_t w[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int k = c * 8 + e * 2;
          const float x = ex2_approx(fmaf(__uint_as_float(r[k >> 5][k & 31]), p.k1, base));
          const float y = ex2_approx(fmaf(__uint_as_float(r[k >> 5][(k & 31) + 1]), p.k1, base));
          l += x + y;
          w[e] = pack_bf16(x, y);
        }
        const int chunk = c ^ (row & 7);  // the copy engine's 128-byte swizzle
        *reinterpret_cast<uint4*>(prow + chunk * 16) = make_uint4(w[0], w[1], w[2], w[3]);
      }
      tc_fence_before();
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[wg]);
    }
    ml[wg][row] = make_float2(ref, l);
  }
  __syncthreads();
  int failed = abort_flag != 0;
  if (!failed) failed = !mbar_wait_bounded(&o_full, 0);
  failed = __syncthreads_or(failed);
  tc_fence_after();
  if (failed) {
    if (tid == 0) atomicOr(p.status, DEV_WAIT_TIMEOUT);
  } else if (warp < 8) {
    const int row = (warp & 3) * 32 + lane;
    const uint32_t base = o_tmem + ((uint32_t)((warp & 3) * 32) << 16);
    const float2 a = ml[0][row], b = ml[1][row];
    const float sink = p.sink ? p.sink[h] * 1.44269504088896340736f : -INFINITY;
    const float top = fmaxf(fmaxf(a.x, b.x), sink);
    const float ca = exp2f(a.x - top), cb = b.x == -INFINITY ? 0.f : exp2f(b.x - top);
    const float inv = 1.0f / (a.y * ca + b.y * cb + exp2f(sink - top));
    const float wa = ca * inv, wb = cb * inv;
    const bool two = n_tiles > 1;
    const int64_t at = (int64_t)(tile.row0 + row) * p.out_ld + (int64_t)h * p.v_dim;
    for (int c = (warp >> 2) * 16; c < p.nv; c += 32) {
      uint32_t x[16], y[16];
      tmem_ld16(base + c, x);
      if (two) tmem_ld16(base + p.o_step + c, y);
      if ((uint32_t)row < tile.rows) {
        float v[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          v[e] = __uint_as_float(x[e]) * wa;
          if (two) v[e] = fmaf(__uint_as_float(y[e]), wb, v[e]);
        }
        bf16* o = p.out + at + c;
        if (c + 16 <= p.v_dim && (reinterpret_cast<uintptr_t>(o) & 15u) == 0) {
          uint32_t w[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) w[e] = pack_bf16(v[2 * e], v[2 * e + 1]);
          reinterpret_cast<uint4*>(o)[0] = make_uint4(w[0], w[1], w[2], w[3]);
          reinterpret_cast<uint4*>(o)[1] = make_uint4(w[4], w[5], w[6], w[7]);
        } else {
#pragma unroll
          for (int e = 0; e < 16; ++e)
            if (c + e < p.v_dim) o[e] = to_elem<bf16>(v[e]);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 9) tmem_dealloc(tmem, p.tmem_cols);
}

// Stages of the two rings and the shared memory they come to; false: two of each do not fit.
static bool softmax_stages(const SoftmaxPrefill& p, int* k_stages, int* v_stages, size_t* smem) {
  const size_t kp = (p.dim + 63) / 64 + (p.rot + 63) / 64, vp = (p.vdim + 63) / 64;
  const size_t fixed = 1024 + kp * SX_Q * 128 + 2 * SX_P_BYTES, one = (size_t)SX_K * 128;
  int k = SX_MAX_STAGES, v = SX_MAX_STAGES;
  while (k > 2 && fixed + one * (k * kp + v * vp) > 222 * 1024) k >= v ? --k : --v;
  if (k == 2) v = std::min(v, 2);
  *k_stages = k;
  *v_stages = v;
  *smem = fixed + one * (k * kp + v * vp);
  return *smem <= 222 * 1024;
}

bool softmax_prefill_fits(const SoftmaxPrefill& p) {
  int k = 0, v = 0;
  size_t smem = 0;
  return p.dim && p.vdim && p.vdim <= 192 && p.n_tiles <= 65535 && p.scale > 0.f &&
         p.keys < (1 << 30) && softmax_stages(p, &k, &v, &smem) && tm_encoder();
}

int32_t launch_softmax_prefill(kanso_cuda_ctx* ctx, const SoftmaxPrefill& p, bool* handled) {
  *handled = false;
  if (!softmax_prefill_fits(p)) return KANSO_OK;
  TmEncodeFn encode = tm_encoder();
  SoftmaxArgs a;
  a.tiles = p.tiles;
  a.sink = p.sink;
  a.out = p.out;
  a.out_ld = p.out_ld;
  a.k1 = p.scale * 1.44269504088896340736f;
  a.v_dim = (int)p.vdim;
  a.nv = (int)((p.vdim + 15u) & ~15u);
  a.o_step = (a.nv + 31) & ~31;
  a.k_panels = (int)((p.dim + 63u) / 64u);
  a.r_panels = (int)((p.rot + 63u) / 64u);
  a.v_panels = (int)((p.vdim + 63u) / 64u);
  a.k_steps = (int)((p.dim + 15u) / 16u);
  a.r_steps = (int)((p.rot + 15u) / 16u);
  a.tmem_cols = 2 * SX_K + 2 * a.o_step <= 256 ? 256 : 512;
  a.status = ctx->dev_status;
  size_t smem = 0;
  softmax_stages(p, &a.k_stages, &a.v_stages, &smem);
  const uint64_t dl = round_up8(p.dim), vl = round_up8(p.vdim), rl = round_up8(p.rot), H = p.heads;
  CUtensorMap qm, qrm, km, krm, vm;
  bool ok = tm_map3(encode, p.q, dl, H, (uint64_t)p.q_rows, dl, H * dl, 1, SX_Q, &qm) &&
            tm_map3(encode, p.k, dl, H, (uint64_t)p.keys, dl, (uint64_t)p.k_ld, 1, SX_K, &km) &&
            tm_map3(encode, p.v, vl, H, (uint64_t)p.keys, vl, (uint64_t)p.v_ld, 1, SX_K, &vm);
  qrm = qm;
  krm = km;
  if (ok && p.rot)
    ok = tm_map3(encode, p.q_rot, rl, H, (uint64_t)p.q_rows, rl, H * rl, 1, SX_Q, &qrm) &&
         tm_map2(encode, p.k_rot, rl, (uint64_t)p.keys, rl, SX_K, &krm);
  if (!ok) return KANSO_OK;
  int32_t st = allow_max_smem(ctx, (const void*)softmax_prefill_kernel);
  if (st) return st;
  *handled = true;
  const cudaError_t e = launch_dependent(ctx, softmax_prefill_kernel, dim3(p.heads, p.n_tiles),
                                         dim3(SX_THREADS), smem, qm, qrm, km, krm, vm, a);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "softmax prefill launch");
  return after_launch(ctx, "softmax_prefill");
}

}  // namespace kanso
