// Prompt attention with sigmoid weights on tcgen05 (bfloat16): 128 query rows of one head against
// key tiles of 64, scores and the output accumulator in TMEM.
//
// Because the weights are not normalised over keys there is no running maximum and nothing to
// rescale: the output is one accumulator that every tile's weights x values product adds to.
//
//   warp 8     copies: a tile's pages by tensor map, one box per page and 64 columns, into a
//              two-stage ring (128-byte swizzle); page numbers are looked up in the block table
//   warp 9     issues S = Q K^T (M = 128, N = 64) into one of two score buffers and O += P V
//              (V as it lies in the pool, N-major) from the tile before
//   warps 0-7  two groups of four, one per score buffer: a thread owns a query row, reads its
//              scores from TMEM, forms the weights and writes them as the bfloat16 A operand P
//
// The distance term, the head's constant and the mask come from one table in shared memory,
// tab[d] = -log2(e) * (cap + pb - r1 ln(1 + r2 d)) for visible distances and +infinity for the
// others, so that a masked weight is 1 / (1 + 2^inf) = 0 without a comparison.
#include <algorithm>

#include "dense.cuh"
#include "tc05.cuh"
#include "tensor_map.h"
#include "warp_mma.cuh"

namespace kanso {

constexpr int SP_Q = 128, SP_K = 64, SP_STAGES = 2;
constexpr int SP_WORKERS = 256, SP_THREADS = 320;
constexpr int SP_TAB_BELOW = 192, SP_TAB_ABOVE = 208;  // masked entries at the table's two ends
constexpr uint32_t SP_MAX_WINDOW = 8192;
constexpr int SP_P_BYTES = SP_Q * SP_K * 2;

struct PrefillArgs {
  SigmoidAttn a;
  const uint32_t* tables;
  const AttnTile* tiles;
  void* out;
  int64_t out_ld;
  uint32_t max_blocks, num_blocks, block_size, kv_heads, group;
  int out_f32, v_dim, nv;        // nv: v_dim rounded up to 16
  int k_panels, v_panels, k_steps;  // 64-column panels of K and V; 16-column steps of the scores
  int tab_n;
  uint32_t tmem_cols;
  int* status;
};

__global__ void __launch_bounds__(SP_THREADS, 1)
    sigmoid_prefill_kernel(const __grid_constant__ CUtensorMap qmap,
                           const __grid_constant__ CUtensorMap kmap,
                           const __grid_constant__ CUtensorMap vmap, const PrefillArgs p) {
  extern __shared__ uint8_t raw[];
  __shared__ uint64_t q_full, k_full[SP_STAGES], k_empty[SP_STAGES], v_full[SP_STAGES],
      v_empty[SP_STAGES], s_full[2], s_free[2], p_full[2], p_free[2], o_full;
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, g = h / (int)p.group;
  const uint32_t k_bytes = (uint32_t)p.k_panels * SP_K * 128u;
  const uint32_t v_bytes = (uint32_t)p.v_panels * SP_K * 128u;
  const uint32_t q_panel = SP_Q * 128u;
  uint8_t* Qs = raw + ((1024u - (smem_u32(raw) & 1023u)) & 1023u);
  uint8_t* Ks = Qs + (size_t)p.k_panels * q_panel;
  uint8_t* Vs = Ks + (size_t)SP_STAGES * k_bytes;
  uint8_t* Ps = Vs + (size_t)SP_STAGES * v_bytes;
  float* tab = reinterpret_cast<float*>(Ps + 2 * SP_P_BYTES);  // [below + window + above]

  pdl_launch_dependents();
  if (tid == 0) {
    mbar_init(&q_full, 1);
    mbar_init(&o_full, 1);
    for (int i = 0; i < SP_STAGES; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_free[i], SP_WORKERS / 2);
      mbar_init(&p_full[i], SP_WORKERS / 2);
      mbar_init(&p_free[i], 1);
    }
    mbar_fence_init();
    abort_flag = 0;
  }
  const float cap = p.a.softcap;
  const float L2E = 1.44269504088896340736f;
  for (int i = tid; i < p.tab_n; i += SP_THREADS) {
    const int d = i - SP_TAB_BELOW;
    tab[i] = d >= 0 && d < (int)p.a.window
                 ? -L2E * (cap + p.a.bias[(size_t)h * p.a.bias_len + d])
                 : INFINITY;
  }
  const AttnTile tile = p.tiles[blockIdx.x];
  const uint32_t q_end = tile.pos0 + tile.rows;  // exclusive
  const uint32_t lo = tile.pos0 + 1 > p.a.window ? tile.pos0 + 1 - p.a.window : 0;
  const uint32_t k_begin = lo / p.block_size * p.block_size;  // tiles start on a page
  const int n_tiles = (int)((q_end - k_begin + SP_K - 1) / SP_K);
  // TMEM only once the kernels in front have ended: they may hold or still want some of it
  pdl_wait();
  if (warp == 9) tmem_alloc(&tmem_slot, p.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot, o_tmem = tmem + 2 * SP_K;

  if (warp == 8) {
    // ---- copies ----
    const int pages = SP_K / (int)p.block_size;  // at most eight
    const uint32_t last_page = (q_end - 1) / p.block_size;
    const uint32_t* table = p.tables + (size_t)tile.seq * p.max_blocks;
    if (lane == 0) {
      mbar_arrive_expect_tx(&q_full, (uint32_t)p.k_panels * q_panel);
      for (int c = 0; c < p.k_panels; ++c)
        tma_load_3d(Qs + (size_t)c * q_panel, &qmap, c * 64, h, (int)tile.row0, &q_full);
    }
    auto page_of = [&](int i) {
      // pages past the last token hold no visible key: the last one stands in for them
      const uint32_t pg =
          min(k_begin / p.block_size + (uint32_t)(i * pages + min(lane, pages - 1)), last_page);
      uint32_t b = table[pg];
      if (b >= p.num_blocks) {
        atomicOr(p.status, DEV_BAD_INDEX);
        b = 0;
      }
      return b;
    };
    uint32_t block = page_of(0);
    int issued = 0;
    for (int i = 0; i < n_tiles; ++i) {
      const int s = i % SP_STAGES;
      const uint32_t par = ((uint32_t)(i / SP_STAGES) & 1u) ^ 1u;
      const uint32_t next = i + 1 < n_tiles ? page_of(i + 1) : 0u;
      bool ok = mbar_wait_abort(&k_empty[s], par, &abort_flag);
      if (lane == 0 && ok) mbar_arrive_expect_tx(&k_full[s], k_bytes);
      __syncwarp();
      ok = __all_sync(0xFFFFFFFFu, ok);
      if (!ok) break;
      const int rec = (int)(block * p.kv_heads + (uint32_t)g);
      if (lane < pages)
        for (int c = 0; c < p.k_panels; ++c)
          tma_load_3d(Ks + (size_t)s * k_bytes + (size_t)c * SP_K * 128 +
                          (size_t)lane * p.block_size * 128,
                      &kmap, c * 64, 0, rec, &k_full[s]);
      ok = mbar_wait_abort(&v_empty[s], par, &abort_flag);
      if (lane == 0 && ok) mbar_arrive_expect_tx(&v_full[s], v_bytes);
      __syncwarp();
      ok = __all_sync(0xFFFFFFFFu, ok);
      if (ok && lane < pages)
        for (int c = 0; c < p.v_panels; ++c)
          tma_load_3d(Vs + (size_t)s * v_bytes + (size_t)c * SP_K * 128 +
                          (size_t)lane * p.block_size * 128,
                      &vmap, c * 64, 0, rec, &v_full[s]);
      issued = i + 1;
      if (!ok) break;
      block = next;
    }
    // leave only when every copy has landed (bounded)
    if (lane == 0) {
      mbar_wait_bounded(&q_full, 0);
      for (int i = max(0, issued - SP_STAGES); i < issued; ++i) {
        mbar_wait_bounded(&k_full[i % SP_STAGES], (uint32_t)(i / SP_STAGES) & 1u);
        if (!abort_flag) mbar_wait_bounded(&v_full[i % SP_STAGES], (uint32_t)(i / SP_STAGES) & 1u);
      }
    }
    __syncwarp();
  } else if (warp == 9) {
    // ---- products ----
    if (lane == 0) {
      const uint32_t id_s = tc_idesc_bf16(SP_Q, SP_K);
      const uint32_t id_o = tc_idesc_bf16(SP_Q, p.nv) | (1u << 16);  // B is N-major
      bool ok = mbar_wait_abort(&q_full, 0, &abort_flag);
      auto scores = [&](int i) {
        const int s = i % SP_STAGES;
        if (ok) ok = mbar_wait_abort(&k_full[s], (uint32_t)(i / SP_STAGES) & 1u, &abort_flag);
        if (!ok) return;
        tc_fence_after();
        for (int k = 0; k < p.k_steps; ++k) {
          const uint32_t panel = (uint32_t)k >> 2, in = ((uint32_t)k & 3u) * 2u;
          const uint64_t ad = tc_smem_desc_sw128(smem_u32(Qs) + panel * q_panel) + in;
          const uint64_t bd =
              tc_smem_desc_sw128(smem_u32(Ks) + (uint32_t)s * k_bytes + panel * (SP_K * 128u)) + in;
          tc_mma_f16(tmem + (uint32_t)(i & 1) * SP_K, ad, bd, id_s, k > 0);
        }
        tc_commit(&k_empty[s]);
        tc_commit(&s_full[i & 1]);
      };
      scores(0);
      if (n_tiles > 1) scores(1);
      for (int i = 0; i < n_tiles && ok; ++i) {
        const int b = i & 1, s = i % SP_STAGES;
        const uint32_t par = (uint32_t)(i >> 1) & 1u;
        if (i + 2 < n_tiles) {
          ok = mbar_wait_abort(&s_free[b], par, &abort_flag);
          if (!ok) break;
          tc_fence_after();
          scores(i + 2);
        }
        if (ok) ok = mbar_wait_abort(&v_full[s], (uint32_t)(i / SP_STAGES) & 1u, &abort_flag);
        if (ok) ok = mbar_wait_abort(&p_full[b], par, &abort_flag);
        if (!ok) break;
        tc_fence_after();
        const uint64_t ad = tc_smem_desc_sw128(smem_u32(Ps) + (uint32_t)b * SP_P_BYTES);
        const uint64_t bd =
            tc_smem_desc_nmajor(smem_u32(Vs) + (uint32_t)s * v_bytes, SP_K * 128u);
#pragma unroll
        for (int k = 0; k < SP_K / 16; ++k)
          tc_mma_f16(o_tmem, ad + 2 * k, bd + 128 * k, id_o, (i > 0 || k > 0) ? 1u : 0u);
        tc_commit(&v_empty[s]);
        tc_commit(&p_free[b]);
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
    const uint32_t s_lane = tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)wg * SP_K;
    uint8_t* prow = Ps + (size_t)wg * SP_P_BYTES + (size_t)row * 128;
    const float k1 = cap != 0.f ? p.a.scale * 2.f * L2E / cap : 0.f;
    const float c1 = 2.f * cap * L2E, k0s = -L2E * p.a.scale;
    for (int i = wg; i < n_tiles; i += 2) {
      const uint32_t par = (uint32_t)(i >> 1) & 1u;
      if (!mbar_wait_abort(&s_full[wg], par, &abort_flag)) break;
      if (!mbar_wait_abort(&p_free[wg], par ^ 1u, &abort_flag)) break;
      __syncwarp();
      tc_fence_after();
      // tab index of the tile's first key; it falls by one per key
      const float* tb = tab + ((int)(tile.pos0 + row) - (int)(k_begin + (uint32_t)i * SP_K) +
                               SP_TAB_BELOW);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t r[32];
        tmem_ld32(s_lane + half * 32, r);
        if (half == 1) {
          tc_fence_before();
          mbar_arrive(&s_free[wg]);
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t w[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float v[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              const int col = c * 8 + e * 2 + u;
              const float s = __uint_as_float(r[col]), b = tb[-(half * 32 + col)];
              const float arg = cap != 0.f ? fmaf(rcp_approx(1.f + ex2_approx(s * k1)), c1, b)
                                           : fmaf(s, k0s, b);
              v[u] = rcp_approx(1.f + ex2_approx(arg));
            }
            const __nv_bfloat162 pk = __floats2bfloat162_rn(v[0], v[1]);
            w[e] = *reinterpret_cast<const uint32_t*>(&pk);
          }
          const int chunk = (half * 4 + c) ^ (row & 7);  // the copy engine's 128-byte swizzle
          *reinterpret_cast<uint4*>(prow + chunk * 16) = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
      fence_proxy_async_smem();
      mbar_arrive(&p_full[wg]);
    }
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
    const int64_t at = (int64_t)(tile.row0 + row) * p.out_ld + (int64_t)h * p.v_dim;
    for (int c = (warp >> 2) * 16; c < p.nv; c += 32) {
      uint32_t r[16];
      tmem_ld16(base + c, r);
      if ((uint32_t)row < tile.rows) {
        if (p.out_f32) {
          float* o = static_cast<float*>(p.out) + at + c;
#pragma unroll
          for (int e = 0; e < 16; ++e)
            if (c + e < p.v_dim) o[e] = __uint_as_float(r[e]);
        } else {
          bf16* o = static_cast<bf16*>(p.out) + at + c;
          if (c + 16 <= p.v_dim && (reinterpret_cast<uintptr_t>(o) & 15u) == 0) {
            uint32_t w[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) {
              const __nv_bfloat162 pk = __floats2bfloat162_rn(__uint_as_float(r[2 * e]),
                                                              __uint_as_float(r[2 * e + 1]));
              w[e] = *reinterpret_cast<const uint32_t*>(&pk);
            }
            reinterpret_cast<uint4*>(o)[0] = make_uint4(w[0], w[1], w[2], w[3]);
            reinterpret_cast<uint4*>(o)[1] = make_uint4(w[4], w[5], w[6], w[7]);
          } else {
#pragma unroll
            for (int e = 0; e < 16; ++e)
              if (c + e < p.v_dim) o[e] = to_elem<bf16>(__uint_as_float(r[e]));
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 9) tmem_dealloc(tmem, p.tmem_cols);
}

int32_t launch_sigmoid_attn_prefill(kanso_cuda_ctx* ctx, const SigmoidAttn& a,
                                    const KvDenseLayer& kv, const void* q, int64_t q_rows,
                                    const RowMap& map, const AttnTile* tiles, uint32_t n_tiles,
                                    void* out, bool out_f32, int64_t out_ld, bool* handled) {
  *handled = false;
  TmEncodeFn encode = tm_encoder();
  const uint32_t bs = kv.block_size;
  if (!encode || kv.k_dim > 256 || kv.v_dim > 256 || a.heads > 65535 || !a.window ||
      a.window > std::min(a.bias_len, SP_MAX_WINDOW) || (bs != 8 && bs != 16 && bs != 32 && bs != 64))
    return KANSO_OK;
  PrefillArgs p;
  p.a = a;
  p.tables = map.tables;
  p.tiles = tiles;
  p.out = out;
  p.out_ld = out_ld;
  p.max_blocks = map.max_blocks;
  p.num_blocks = kv.num_blocks;
  p.block_size = bs;
  p.kv_heads = kv.kv_heads;
  p.group = a.heads / kv.kv_heads;
  p.out_f32 = out_f32;
  p.v_dim = (int)kv.v_dim;
  p.nv = (int)((kv.v_dim + 15u) & ~15u);
  p.k_panels = (int)((kv.k_dim + 63u) / 64u);
  p.v_panels = (int)((kv.v_dim + 63u) / 64u);
  p.k_steps = (int)((kv.k_dim + 15u) / 16u);
  p.tab_n = SP_TAB_BELOW + (int)a.window + SP_TAB_ABOVE;
  p.tmem_cols = 2 * SP_K + p.nv <= 256 ? 256 : 512;
  p.status = ctx->dev_status;
  const size_t smem = 1024 + (size_t)p.k_panels * SP_Q * 128 +
                      (size_t)SP_STAGES * SP_K * 128 * (p.k_panels + p.v_panels) +
                      2 * (size_t)SP_P_BYTES + (size_t)p.tab_n * 4;
  if (smem > 225 * 1024) return KANSO_OK;
  const uint64_t records = (uint64_t)kv.num_blocks * kv.kv_heads;
  CUtensorMap qm, km, vm;
  const bf16* pool = reinterpret_cast<const bf16*>(kv.base);
  if (!tm_map3(encode, q, kv.k_ld, a.heads, (uint64_t)q_rows, kv.k_ld, (uint64_t)a.heads * kv.k_ld, 1,
            SP_Q, &qm) ||
      !tm_map3(encode, pool, kv.k_ld, bs, records, kv.k_ld, kv.rec_elems, bs, 1, &km) ||
      !tm_map3(encode, pool + (size_t)bs * kv.k_ld, kv.v_ld, bs, records, kv.v_ld, kv.rec_elems, bs, 1,
            &vm))
    return KANSO_OK;
  int32_t st = allow_max_smem(ctx, (const void*)sigmoid_prefill_kernel);
  if (st) return st;
  *handled = true;
  const cudaError_t e = launch_dependent(ctx, sigmoid_prefill_kernel, dim3(n_tiles, a.heads),
                                         dim3(SP_THREADS), smem, qm, km, vm, p);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "sigmoid prefill launch");
  return after_launch(ctx, "sigmoid_prefill");
}

}  // namespace kanso
