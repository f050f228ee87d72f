// Matrix memory with exponential gates. Per head, from S = 0, n = 0, m = 0:
//
//   i = cap tanh((W_i h + b_i) / cap)             f = log sigmoid(cap tanh((W_f h + b_f) / cap))
//   m' = max(f + m, i)
//   S' = exp(f + m - m') S + exp(i - m') k v^T    n' likewise with k alone
//   o = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6)                    q scaled by dim^-1/2
//
// Everything but the products of the chunk form is f32. The state lies in records of 32 value
// columns with their own n and m (KvStateLayer), so a CTA needs nothing of another.
//
// mlstm_step: one token per sequence; the state streams through registers, requested before the
// wait for the projections in front. mlstm_rows: portions token by token with the state in shared
// memory. mlstm_chunk: prompts, 64 tokens at a time on the tensor cores.
//
// The chunk form. With F_t = f_1 + ... + f_t inside the chunk, u_j = i_j - F_j and
// G_t = max(m, u_1, ..., u_t) the maximum is m_t = F_t + G_t, and
//
//   o_t ~ sum_{j <= t} exp(u_j - G_t) (q_t . k_j) v_j + exp(m - G_t) S^T q_t
//   S'  = exp(m - G_L) S + sum_j exp(u_j - G_L) k_j v_j^T
//
// all exponents <= 0. q, k and v are bfloat16 values (projections); every f32 factor that meets
// them in a product (weights, state, decayed values) goes in as the sum of two bfloat16 values, so
// that the products keep about 16 bits of it.
#include <algorithm>
#include <cmath>

#include "dense.cuh"
#include "warp_mma.cuh"

namespace kanso {

constexpr int ML_THREADS = 256;
constexpr int ML_COLS = KvStateLayer::kCols;

__device__ __forceinline__ float ml_value(const MlstmArgs& a, int64_t at) {
  float v = a.y[at];
  for (int p = 1; p < a.parts; ++p) v += a.y[p * a.part_stride + at];
  return v;
}
__device__ __forceinline__ float ml_input_gate(const MlstmArgs& a, const int64_t row, int h) {
  const int64_t at = row * a.width() + (int64_t)a.heads * (2 * a.dim + 2 * a.vdim) + h;
  return a.cap * tanhf((ml_value(a, at) + a.i_bias[h]) / a.cap);
}
__device__ __forceinline__ float ml_forget_gate(const MlstmArgs& a, const int64_t row, int h) {
  const int64_t at = row * a.width() + (int64_t)a.heads * (2 * a.dim + 2 * a.vdim + 1) + h;
  const float z = a.cap * tanhf((ml_value(a, at) + a.f_bias[h]) / a.cap);
  return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));  // log sigmoid
}
struct MlPortion {
  int64_t row0;
  uint32_t rows, pos0, slot;
};
__device__ __forceinline__ MlPortion ml_portion(const MlstmArgs& a, uint32_t i) {
  MlPortion p;
  uint32_t seq = i;
  if (a.portions) {
    const AttnTile t = a.portions[i];
    p.row0 = t.row0, p.rows = t.rows, p.pos0 = t.pos0;
    seq = t.seq;
  } else {
    p.row0 = i, p.rows = 1, p.pos0 = a.positions[i];
  }
  p.slot = a.slots ? a.slots[seq] : seq;
  return p;
}

// Sums over the CTA of a float4 of column group tid % 8: column c of the sums in out[c].
__device__ __forceinline__ void ml_column_sums(float4 v, float (*red)[ML_COLS], float* out) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 8; o < 32; o <<= 1) {
    v.x += __shfl_xor_sync(0xFFFFFFFFu, v.x, o);
    v.y += __shfl_xor_sync(0xFFFFFFFFu, v.y, o);
    v.z += __shfl_xor_sync(0xFFFFFFFFu, v.z, o);
    v.w += __shfl_xor_sync(0xFFFFFFFFu, v.w, o);
  }
  if (lane < 8) *reinterpret_cast<float4*>(&red[warp][lane * 4]) = v;
  __syncthreads();
  if (threadIdx.x < ML_COLS) {
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < ML_THREADS / 32; ++w) s += red[w][threadIdx.x];
    out[threadIdx.x] = s;
  }
  __syncthreads();
}

// ------------------------------------------------------------- one token per sequence ----
// A thread owns four columns of every 32nd row of its tile, AHEAD of them at a time.
template <int AHEAD>
__global__ void __launch_bounds__(ML_THREADS) mlstm_step_kernel(const MlstmArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(16) float red[ML_THREADS / 32][ML_COLS], vs[ML_COLS], os[ML_COLS];
  __shared__ float sums[32], gate[2];
  const int tid = threadIdx.x, tile = blockIdx.x, h = blockIdx.y;
  const int D = a.dim, V = a.vdim, H = a.heads;
  float *qs = sm, *ks = sm + D;
  pdl_launch_dependents();
  const MlPortion p = ml_portion(a, blockIdx.z);
  const bool fresh = p.pos0 == 0;
  float* rec = a.state.at(p.slot, h, tile);
  float* nst = rec + a.state.n_at();
  const int c4 = (tid & 7) * 4, r0 = tid >> 3;
  float4 s[AHEAD];
  // the state was written by an earlier step
  auto fetch = [&](int first) {
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int r = first + i * 32;
      s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && r < D) s[i] = __ldcs(reinterpret_cast<const float4*>(rec + r * ML_COLS + c4));
    }
  };
  fetch(r0);
  const float m = fresh ? 0.f : rec[a.state.m_at()];
  pdl_wait();
  const int64_t row = p.row0 * a.width();
  const float scale = 1.0f / sqrtf((float)D);
  for (int i = tid; i < D; i += ML_THREADS) {
    qs[i] = ml_value(a, row + (int64_t)h * D + i) * scale;
    ks[i] = ml_value(a, row + (int64_t)(H + h) * D + i);
  }
  if (tid < ML_COLS) {
    const int c = tile * ML_COLS + tid;
    vs[tid] = c < V ? ml_value(a, row + (int64_t)2 * H * D + (int64_t)h * V + c) : 0.f;
  }
  if (tid == 64) gate[0] = ml_input_gate(a, p.row0, h);
  if (tid == 96) gate[1] = ml_forget_gate(a, p.row0, h);
  __syncthreads();
  const float ig = gate[0], fg = gate[1];
  const float m1 = fmaxf(fg + m, ig), keep = expf(fg + m - m1), take = expf(ig - m1);
  const float4 v = *reinterpret_cast<const float4*>(vs + c4);
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int first = r0; first < D; first += AHEAD * 32) {
    if (first != r0) fetch(first);
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int r = first + i * 32;
      if (r >= D) continue;
      const float k = take * ks[r], q = qs[r];
      float4 x = s[i];
      x.x = fmaf(keep, x.x, k * v.x), x.y = fmaf(keep, x.y, k * v.y);
      x.z = fmaf(keep, x.z, k * v.z), x.w = fmaf(keep, x.w, k * v.w);
      o.x = fmaf(q, x.x, o.x), o.y = fmaf(q, x.y, o.y);
      o.z = fmaf(q, x.z, o.z), o.w = fmaf(q, x.w, o.w);
      __stcs(reinterpret_cast<float4*>(rec + r * ML_COLS + c4), x);
    }
  }
  float nq = 0.f;
  for (int i = tid; i < D; i += ML_THREADS) {
    const float n = fmaf(keep, fresh ? 0.f : nst[i], take * ks[i]);
    nst[i] = n;
    nq = fmaf(n, qs[i], nq);
  }
  nq = block_sum(nq, sums);
  ml_column_sums(o, red, os);
  if (tid == 0) rec[a.state.m_at()] = m1;
  const float den = fmaxf(fabsf(nq), expf(-m1)) + 1e-6f;
  const int c = tile * ML_COLS + tid;
  if (tid < ML_COLS && c < V) a.out[p.row0 * H * V + (int64_t)h * V + c] = os[tid] / den;
}

// ------------------------------------------------------------- portions token by token ----
__global__ void __launch_bounds__(ML_THREADS) mlstm_rows_kernel(const MlstmArgs a, int in_smem) {
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(16) float red[ML_THREADS / 32][ML_COLS], vs[ML_COLS], os[ML_COLS];
  __shared__ float sums[32], gate[2];
  const int tid = threadIdx.x, tile = blockIdx.x, h = blockIdx.y;
  const int D = a.dim, V = a.vdim, H = a.heads, D4 = (D + 3) & ~3;
  float *qs = sm, *ks = qs + D4, *ns = ks + D4;
  pdl_launch_dependents();
  pdl_wait();
  const MlPortion p = ml_portion(a, blockIdx.z);
  float* rec = a.state.at(p.slot, h, tile);
  float* S = in_smem ? ns + D4 : rec;  // [D][32]
  const bool fresh = p.pos0 == 0;
  for (int i = tid; i < D * ML_COLS; i += ML_THREADS)
    if (in_smem || fresh) S[i] = fresh ? 0.f : rec[i];
  for (int i = tid; i < D; i += ML_THREADS) ns[i] = fresh ? 0.f : rec[a.state.n_at() + i];
  float m = fresh ? 0.f : rec[a.state.m_at()];
  const int c4 = (tid & 7) * 4, r0 = tid >> 3;
  const float scale = 1.0f / sqrtf((float)D);
  for (uint32_t t = 0; t < p.rows; ++t) {
    const int64_t row = (p.row0 + t) * a.width();
    __syncthreads();
    for (int i = tid; i < D; i += ML_THREADS) {
      qs[i] = ml_value(a, row + (int64_t)h * D + i) * scale;
      ks[i] = ml_value(a, row + (int64_t)(H + h) * D + i);
    }
    if (tid < ML_COLS) {
      const int c = tile * ML_COLS + tid;
      vs[tid] = c < V ? ml_value(a, row + (int64_t)2 * H * D + (int64_t)h * V + c) : 0.f;
    }
    if (tid == 64) gate[0] = ml_input_gate(a, p.row0 + t, h);
    if (tid == 96) gate[1] = ml_forget_gate(a, p.row0 + t, h);
    __syncthreads();
    const float ig = gate[0], fg = gate[1];
    const float m1 = fmaxf(fg + m, ig), keep = expf(fg + m - m1), take = expf(ig - m1);
    m = m1;
    const float4 v = *reinterpret_cast<const float4*>(vs + c4);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int r = r0; r < D; r += 32) {
      const float k = take * ks[r], q = qs[r];
      float4 x = *reinterpret_cast<const float4*>(S + r * ML_COLS + c4);
      x.x = fmaf(keep, x.x, k * v.x), x.y = fmaf(keep, x.y, k * v.y);
      x.z = fmaf(keep, x.z, k * v.z), x.w = fmaf(keep, x.w, k * v.w);
      o.x = fmaf(q, x.x, o.x), o.y = fmaf(q, x.y, o.y);
      o.z = fmaf(q, x.z, o.z), o.w = fmaf(q, x.w, o.w);
      *reinterpret_cast<float4*>(S + r * ML_COLS + c4) = x;
    }
    float nq = 0.f;
    for (int i = tid; i < D; i += ML_THREADS) {
      const float n = fmaf(keep, ns[i], take * ks[i]);
      ns[i] = n;
      nq = fmaf(n, qs[i], nq);
    }
    nq = block_sum(nq, sums);
    ml_column_sums(o, red, os);
    const float den = fmaxf(fabsf(nq), expf(-m)) + 1e-6f;
    const int c = tile * ML_COLS + tid;
    if (tid < ML_COLS && c < V)
      a.out[(p.row0 + t) * H * V + (int64_t)h * V + c] = os[tid] / den;
  }
  __syncthreads();
  if (in_smem)
    for (int i = tid; i < D * ML_COLS; i += ML_THREADS) rec[i] = S[i];
  for (int i = tid; i < D; i += ML_THREADS) rec[a.state.n_at() + i] = ns[i];
  if (tid == 0) rec[a.state.m_at()] = m;
}

// ------------------------------------------------------------- prompts in chunks ----
// The operands in bfloat16, rows of 16-byte multiples: q, k [T][heads][dim ld], v [T][heads][vdim
// ld]; gates f32 [T][heads].
struct MlOperands {
  bf16 *q, *k, *v;
  float *ig, *fg;
  int dl, vl;
};

__global__ void __launch_bounds__(ML_THREADS) mlstm_operands_kernel(const MlstmArgs a,
                                                                   const MlOperands w) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x, row = t * a.width();
  const int H = a.heads, D = a.dim, V = a.vdim;
  auto copy = [&](int64_t from, bf16* to, int n, int ld) {
    for (int i = threadIdx.x * 2; i < H * ld; i += ML_THREADS * 2) {
      const int h = i / ld, d = i - h * ld;
      const float x = d < n ? ml_value(a, from + (int64_t)h * n + d) : 0.f;
      const float y = d + 1 < n ? ml_value(a, from + (int64_t)h * n + d + 1) : 0.f;
      *reinterpret_cast<__nv_bfloat162*>(to + t * H * ld + i) = __floats2bfloat162_rn(x, y);
    }
  };
  copy(row, w.q, D, w.dl);
  copy(row + (int64_t)H * D, w.k, D, w.dl);
  copy(row + (int64_t)2 * H * D, w.v, V, w.vl);
  for (int h = threadIdx.x; h < H; h += ML_THREADS) {
    w.ig[t * H + h] = ml_input_gate(a, t, h);
    w.fg[t * H + h] = ml_forget_gate(a, t, h);
  }
}

__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(x, y);
  hi = *reinterpret_cast<const uint32_t*>(&a);
  lo = pack_bf16(x - __bfloat162float(a.x), y - __bfloat162float(a.y));
}

// Eight warps: DW along the state's rows (dim), 8 / DW along its columns, 16 of them each. A warp's
// part of the transposed state, 16 columns x NT * 8 rows, stays in its registers as accumulators,
// whose layout is that of the A operand which S^T Q^T needs.
constexpr int MC_L = 64, MC_PS = MC_L + 8, MC_OS = MC_L + 2;

template <int DW, int NT>
struct McShape {
  static constexpr int kCols = 8 / DW * 16;     // value columns per CTA
  static constexpr int kDim = DW * NT * 8;      // state rows it can hold
  static constexpr int kQs = kDim + 8, kVs = kCols + 8;
  static constexpr size_t kBytes = (size_t)2 * MC_L * kQs * 2 + (size_t)MC_L * kVs * 2 +
                                   (size_t)2 * MC_L * MC_PS * 2 + (size_t)kDim * 4 +
                                   (size_t)(DW - 1) * kCols * MC_OS * 4;
};

template <int DW, int NT>
__global__ void __launch_bounds__(ML_THREADS, 1)
    mlstm_chunk_kernel(const MlstmArgs a, const MlOperands w) {
  using Sh = McShape<DW, NT>;
  constexpr int QS = Sh::kQs, VS = Sh::kVs, COLS = Sh::kCols;
  extern __shared__ __align__(16) uint8_t sm_raw[];
  __shared__ float us[MC_L], gs[MC_L], es[MC_L], as[MC_L], invs[MC_L], dens[2][MC_L], nqs[MC_L],
      fsum[MC_L];
  __shared__ float chunk_m[2];  // G and F at the chunk's end
  bf16* Qs = reinterpret_cast<bf16*>(sm_raw);   // [64][QS]
  bf16* Ks = Qs + MC_L * QS;
  bf16* Vs = Ks + MC_L * QS;                    // [64][VS]
  bf16* Ph = Vs + MC_L * VS;                    // [64][MC_PS], two parts
  bf16* Pl = Ph + MC_L * MC_PS;
  float* ns = reinterpret_cast<float*>(Pl + MC_L * MC_PS);  // [kDim]
  float* Or = ns + Sh::kDim;                                // [DW - 1][COLS][MC_OS]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, H = a.heads, D = a.dim, V = a.vdim;
  const int vw = warp / DW, dw = warp % DW;
  const int col0 = blockIdx.x * COLS;           // the CTA's first value column
  const int quad = lane >> 2, two = (lane & 3) * 2;
  pdl_launch_dependents();
  pdl_wait();
  const MlPortion p = ml_portion(a, blockIdx.z);
  const bool fresh = p.pos0 == 0;

  // the state: columns vw * 16 + quad (+ 8), rows dw * NT * 8 + nt * 8 + two (+ 1)
  float S[NT][4];
  const int vc = vw * 16 + quad;
  auto state_at = [&](int c, int d) -> float* {  // c: column of the CTA
    const int g = col0 + c;
    return a.state.at(p.slot, h, g / ML_COLS) + d * ML_COLS + g % ML_COLS;
  };
  const int tiles = (int)a.state.tiles();
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = vc + (e >> 1) * 8, d = (dw * NT + nt) * 8 + two + (e & 1);
      S[nt][e] = !fresh && d < D && (col0 + c) / ML_COLS < tiles ? *state_at(c, d) : 0.f;
    }
  const float* rec0 = a.state.at(p.slot, h, col0 / ML_COLS);
  for (int i = tid; i < Sh::kDim; i += ML_THREADS)
    ns[i] = !fresh && i < D ? rec0[a.state.n_at() + i] : 0.f;
  float m = fresh ? 0.f : rec0[a.state.m_at()];

  const int dc = Sh::kDim / 8, dlc = w.dl / 8, vlc = w.vl / 8;
  auto fetch_qk = [&](const bf16* src, bf16* dst, uint32_t t0) {
    for (int i = tid; i < MC_L * dc; i += ML_THREADS) {
      const int r = i / dc, c = i - r * dc;
      const bool in = t0 + r < p.rows && c < dlc;
      const bf16* from = src + ((p.row0 + (in ? t0 + r : 0)) * H + h) * w.dl + (in ? c : 0) * 8;
      cp_async16(dst + r * QS + c * 8, from, in);
    }
  };
  auto fetch_v = [&](uint32_t t0) {
    for (int i = tid; i < MC_L * (COLS / 8); i += ML_THREADS) {
      const int r = i / (COLS / 8), c = i % (COLS / 8), g = col0 / 8 + c;
      const bool in = t0 + r < p.rows && g < vlc;
      const bf16* from = w.v + ((p.row0 + (in ? t0 + r : 0)) * H + h) * w.vl + (in ? g : 0) * 8;
      cp_async16(Vs + r * VS + c * 8, from, in);
    }
  };
  fetch_qk(w.q, Qs, 0);
  fetch_qk(w.k, Ks, 0);
  fetch_v(0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  const float scale = 1.0f / sqrtf((float)D);

  for (uint32_t t0 = 0; t0 < p.rows; t0 += MC_L) {
    if (warp == 0) {  // the gates, two tokens per lane
      float f0 = 0.f, f1 = 0.f, i0 = -INFINITY, i1 = -INFINITY;
      const uint32_t t = t0 + lane * 2;
      if (t < p.rows) {
        f0 = w.fg[(p.row0 + t) * H + h];
        i0 = w.ig[(p.row0 + t) * H + h];
      }
      if (t + 1 < p.rows) {
        f1 = w.fg[(p.row0 + t + 1) * H + h];
        i1 = w.ig[(p.row0 + t + 1) * H + h];
      }
      float incl = f0 + f1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xFFFFFFFFu, incl, o);
        if (lane >= o) incl += v;
      }
      const float F1 = incl, F0 = incl - f1;
      const float u0 = i0 - F0, u1 = i1 - F1;
      float top = fmaxf(u0, u1);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xFFFFFFFFu, top, o);
        if (lane >= o) top = fmaxf(top, v);
      }
      float before = __shfl_up_sync(0xFFFFFFFFu, top, 1);
      before = lane ? fmaxf(before, m) : m;
      const float G0 = fmaxf(before, u0), G1 = fmaxf(G0, u1);
      const float GL = __shfl_sync(0xFFFFFFFFu, G1, 31);
      us[lane * 2] = u0, us[lane * 2 + 1] = u1;
      gs[lane * 2] = G0, gs[lane * 2 + 1] = G1;
      es[lane * 2] = expf(m - G0), es[lane * 2 + 1] = expf(m - G1);
      as[lane * 2] = expf(u0 - GL), as[lane * 2 + 1] = expf(u1 - GL);
      fsum[lane * 2] = F0 + G0, fsum[lane * 2 + 1] = F1 + G1;  // the maximum m_t
      if (lane == 31) {
        chunk_m[0] = G1;
        chunk_m[1] = F1;
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // n . q of eight tokens per warp
    for (int r = warp * 8; r < warp * 8 + 8; ++r) {
      float v = 0.f;
      for (int d = lane * 2; d < Sh::kDim; d += 64) {
        float x, y;
        unpack_bf16x2(*reinterpret_cast<const uint32_t*>(Qs + r * QS + d), x, y);
        v = fmaf(x, ns[d], fmaf(y, ns[d + 1], v));
      }
#pragma unroll
      for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
      if (lane == 0) nqs[r] = v * scale;
    }
    // scores of 16 tokens against 32, weighted
    {
      const int mt = (warp & 3) * 16, j0 = (warp >> 2) * 32;
      float c[4][4] = {};
      if (j0 <= mt + 15) {
        const uint32_t qa = smem_u32(Qs) + (uint32_t)((mt + (lane & 15)) * QS + (lane >> 4) * 8) * 2;
        const uint32_t ka = smem_u32(Ks) + (uint32_t)((j0 + (lane & 7) + ((lane >> 4) << 3)) * QS +
                                                      ((lane >> 3) & 1) * 8) * 2;
#pragma unroll 4
        for (int kk = 0; kk < Sh::kDim / 16; ++kk) {
          uint32_t x[4], b[4], d[4];
          ldm_x4(x, qa + kk * 32);
          ldm_x4(b, ka + kk * 32);
          ldm_x4(d, ka + (uint32_t)(16 * QS) * 2 + kk * 32);
          mma_bf16(c[0], x, b[0], b[1]);
          mma_bf16(c[1], x, b[2], b[3]);
          mma_bf16(c[2], x, d[0], d[1]);
          mma_bf16(c[3], x, d[2], d[3]);
        }
      }
      float sum[2] = {0.f, 0.f};
      const float g0 = gs[mt + quad], g1 = gs[mt + quad + 8];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = mt + quad + (e >> 1) * 8, j = j0 + nt * 8 + two + (e & 1);
          const float v = j <= t ? c[nt][e] * scale * expf(us[j] - (e >> 1 ? g1 : g0)) : 0.f;
          c[nt][e] = v;
          sum[e >> 1] += v;
        }
        uint32_t hi, lo;
        const int at = (mt + quad) * MC_PS + j0 + nt * 8 + two;
        split_bf16(c[nt][0], c[nt][1], hi, lo);
        *reinterpret_cast<uint32_t*>(Ph + at) = hi;
        *reinterpret_cast<uint32_t*>(Pl + at) = lo;
        split_bf16(c[nt][2], c[nt][3], hi, lo);
        *reinterpret_cast<uint32_t*>(Ph + at + 8 * MC_PS) = hi;
        *reinterpret_cast<uint32_t*>(Pl + at + 8 * MC_PS) = lo;
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        sum[e] += __shfl_xor_sync(0xFFFFFFFFu, sum[e], 1);
        sum[e] += __shfl_xor_sync(0xFFFFFFFFu, sum[e], 2);
        if ((lane & 3) == 0) dens[warp >> 2][mt + quad + e * 8] = sum[e];
      }
    }
    // S^T Q^T over the warp's rows of the state, 16 columns x 64 tokens
    float o[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    {
      const uint32_t qb = smem_u32(Qs) + (uint32_t)(((lane & 7) + ((lane >> 4) << 3)) * QS +
                                                    ((lane >> 3) & 1) * 8 + dw * NT * 8) * 2;
#pragma unroll
      for (int kk = 0; kk < NT / 2; ++kk) {
        uint32_t hi[4], lo[4];
        split_bf16(S[2 * kk][0], S[2 * kk][1], hi[0], lo[0]);
        split_bf16(S[2 * kk][2], S[2 * kk][3], hi[1], lo[1]);
        split_bf16(S[2 * kk + 1][0], S[2 * kk + 1][1], hi[2], lo[2]);
        split_bf16(S[2 * kk + 1][2], S[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          uint32_t b[4];
          ldm_x4(b, qb + (uint32_t)(nt * 16 * QS + kk * 16) * 2);
          mma_bf16(o[2 * nt], hi, b[0], b[1]);
          mma_bf16(o[2 * nt + 1], hi, b[2], b[3]);
          mma_bf16(o[2 * nt], lo, b[0], b[1]);
          mma_bf16(o[2 * nt + 1], lo, b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float e0 = es[i * 8 + two] * scale, e1 = es[i * 8 + two + 1] * scale;
      o[i][0] *= e0, o[i][1] *= e1, o[i][2] *= e0, o[i][3] *= e1;
    }
    __syncthreads();  // weights and denominators are there, the queries are read out
    if (t0 + MC_L < p.rows) fetch_qk(w.q, Qs, t0 + MC_L);
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (tid < MC_L) {
      const float den = dens[0][tid] + dens[1][tid] + es[tid] * nqs[tid];
      invs[tid] = 1.0f / (fmaxf(fabsf(den), expf(-fsum[tid])) + 1e-6f);
    }
    // the chunk's own tokens: V^T P^T, the keys shared out over the DW warps
    const uint32_t vt = smem_u32(Vs) + (uint32_t)(((lane & 7) + ((lane >> 4) << 3)) * VS + vw * 16 +
                                                  ((lane >> 3) & 1) * 8) * 2;
    {
      const uint32_t pb = (uint32_t)(((lane & 7) + ((lane >> 4) << 3)) * MC_PS +
                                     ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
      for (int kk = dw * (4 / DW); kk < (dw + 1) * (4 / DW); ++kk) {
        uint32_t x[4];
        ldm_x4_t(x, vt + (uint32_t)(kk * 16 * VS) * 2);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          if (nt * 16 + 15 < kk * 16) continue;  // tokens before these keys
          uint32_t b[4], c[4];
          const uint32_t at = pb + (uint32_t)(nt * 16 * MC_PS + kk * 16) * 2;
          ldm_x4(b, smem_u32(Ph) + at);
          ldm_x4(c, smem_u32(Pl) + at);
          mma_bf16(o[2 * nt], x, b[0], b[1]);
          mma_bf16(o[2 * nt + 1], x, b[2], b[3]);
          mma_bf16(o[2 * nt], x, c[0], c[1]);
          mma_bf16(o[2 * nt + 1], x, c[2], c[3]);
        }
      }
    }
    if (dw > 0) {
      float* dst = Or + (size_t)(dw - 1) * COLS * MC_OS;
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; e += 2)
          *reinterpret_cast<float2*>(dst + (vc + e * 4) * MC_OS + i * 8 + two) =
              make_float2(o[i][e], o[i][e + 1]);
    }
    __syncthreads();
    // the results, DW warps per 16 columns share the tokens
    if (dw == 0) {
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int c = vc + (e >> 1) * 8, t = i * 8 + two + (e & 1);
          float v = o[i][e];
#pragma unroll
          for (int k = 0; k < DW - 1; ++k) v += Or[(size_t)(k * COLS + c) * MC_OS + t];
          if (t0 + t < p.rows && col0 + c < V)
            a.out[(p.row0 + t0 + t) * H * V + (int64_t)h * V + col0 + c] = v * invs[t];
        }
    }
    // the state after the chunk
    {
      const float GL = chunk_m[0], keep = expf(m - GL);
      m = chunk_m[1] + GL;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[nt][e] *= keep;
      const uint32_t kb = smem_u32(Ks) + (uint32_t)((lane & 15) * QS + (lane >> 4) * 8 +
                                                    dw * NT * 8) * 2;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t x[4], hi[4], lo[4];
        ldm_x4_t(x, vt + (uint32_t)(kk * 16 * VS) * 2);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          // register i: columns quad (+ 8 for odd i), tokens two, two + 1 (+ 8 for i >= 2)
          const int j = kk * 16 + two + (i >> 1) * 8;
          float v0, v1;
          unpack_bf16x2(x[i], v0, v1);
          split_bf16(v0 * as[j], v1 * as[j + 1], hi[i], lo[i]);
        }
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t b[4];
          ldm_x4_t(b, kb + (uint32_t)(kk * 16 * QS + nt * 8) * 2);
          mma_bf16(S[nt], hi, b[0], b[1]);
          mma_bf16(S[nt + 1], hi, b[2], b[3]);
          mma_bf16(S[nt], lo, b[0], b[1]);
          mma_bf16(S[nt + 1], lo, b[2], b[3]);
        }
      }
      for (int d = tid * 2; d < Sh::kDim; d += ML_THREADS * 2) {
        float x = ns[d] * keep, y = ns[d + 1] * keep;
#pragma unroll 8
        for (int j = 0; j < MC_L; ++j) {
          float k0, k1;
          unpack_bf16x2(*reinterpret_cast<const uint32_t*>(Ks + j * QS + d), k0, k1);
          x = fmaf(as[j], k0, x), y = fmaf(as[j], k1, y);
        }
        ns[d] = x, ns[d + 1] = y;
      }
    }
    __syncthreads();  // keys, values and gates are read out
    if (t0 + MC_L < p.rows) {
      fetch_qk(w.k, Ks, t0 + MC_L);
      fetch_v(t0 + MC_L);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = vc + (e >> 1) * 8, d = (dw * NT + nt) * 8 + two + (e & 1);
      if (d < D && (col0 + c) / ML_COLS < tiles) *state_at(c, d) = S[nt][e];
    }
  for (int g = col0 / ML_COLS; g < min(tiles, (col0 + COLS) / ML_COLS); ++g) {
    float* rec = a.state.at(p.slot, h, g);
    for (int i = tid; i < D; i += ML_THREADS) rec[a.state.n_at() + i] = ns[i];
    if (tid == 0) rec[a.state.m_at()] = m;
  }
}

template <typename... KArgs, typename... Args>
static int32_t ml_launch(kanso_cuda_ctx* ctx, void (*kern)(KArgs...), dim3 grid, size_t smem,
                         const char* what, Args... args) {
  int32_t st = allow_max_smem(ctx, (const void*)kern);
  if (st) return st;
  const cudaError_t e = launch_dependent(ctx, kern, grid, dim3(ML_THREADS), smem, args...);
  if (e != cudaSuccess) return cuda_fail(ctx, e, what);
  return after_launch(ctx, what);
}

static int32_t ml_check(kanso_cuda_ctx* ctx, const MlstmArgs& a, uint32_t n) {
  if (a.heads > 65535 || n > 65535)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "matrix memory: %u heads, %u portions", a.heads, n);
  return KANSO_OK;
}

int32_t launch_mlstm_rows(kanso_cuda_ctx* ctx, const MlstmArgs& a, uint32_t n, uint32_t max_rows) {
  int32_t st = ml_check(ctx, a, n);
  if (st) return st;
  const dim3 grid(a.state.tiles(), a.heads, n);
  if (max_rows == 1) {
    const size_t smem = (size_t)a.dim * 8;
    if (smem <= 200 * 1024) {
      if (a.dim <= 128) return ml_launch(ctx, mlstm_step_kernel<4>, grid, smem, "mlstm_step", a);
      if (a.dim <= 256) return ml_launch(ctx, mlstm_step_kernel<8>, grid, smem, "mlstm_step", a);
      return ml_launch(ctx, mlstm_step_kernel<16>, grid, smem, "mlstm_step", a);
    }
  }
  const size_t rows = (size_t)3 * ((a.dim + 3) & ~3u) * 4, state = (size_t)a.dim * ML_COLS * 4;
  if (rows > 200 * 1024)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "matrix memory: heads of %u columns", a.dim);
  const int in_smem = rows + state <= 200 * 1024;
  return ml_launch(ctx, mlstm_rows_kernel, grid, rows + (in_smem ? state : 0), "mlstm_rows", a,
                   in_smem);
}

bool mlstm_chunk_fits(const MlstmArgs& a) { return a.dim <= 512; }

static size_t ml_room(size_t bytes) { return (bytes + 255) & ~(size_t)255; }
size_t mlstm_chunk_bytes(uint32_t heads, uint32_t dim, uint32_t vdim, int64_t T) {
  const size_t n = (size_t)T * heads;
  return 2 * ml_room(n * round_up8(dim) * 2) + ml_room(n * round_up8(vdim) * 2) +
         2 * ml_room(n * 4);
}

template <int DW, int NT>
static int32_t chunk_launch(kanso_cuda_ctx* ctx, const MlstmArgs& a, const MlOperands& w,
                            uint32_t n) {
  using Sh = McShape<DW, NT>;
  const dim3 grid((a.vdim + Sh::kCols - 1) / Sh::kCols, a.heads, n);
  return ml_launch(ctx, mlstm_chunk_kernel<DW, NT>, grid, Sh::kBytes, "mlstm_chunk", a, w);
}

int32_t launch_mlstm_chunks(kanso_cuda_ctx* ctx, const MlstmArgs& a, uint32_t n, void* mem,
                            int64_t T) {
  int32_t st = ml_check(ctx, a, n);
  if (st) return st;
  MlOperands w;
  w.dl = (int)round_up8(a.dim);
  w.vl = (int)round_up8(a.vdim);
  uint8_t* at = static_cast<uint8_t*>(mem);
  const size_t rows = (size_t)T * a.heads;
  auto take = [&](size_t bytes) {
    uint8_t* r = at;
    at += ml_room(bytes);
    return r;
  };
  w.q = (bf16*)take(rows * w.dl * 2);
  w.k = (bf16*)take(rows * w.dl * 2);
  w.v = (bf16*)take(rows * w.vl * 2);
  w.ig = (float*)take(rows * 4);
  w.fg = (float*)take(rows * 4);
  if ((st = ml_launch(ctx, mlstm_operands_kernel, dim3((unsigned)T), 0, "mlstm_operands", a, w)))
    return st;
  if (a.dim <= 64) return chunk_launch<2, 4>(ctx, a, w, n);
  if (a.dim <= 128) return chunk_launch<2, 8>(ctx, a, w, n);
  if (a.dim <= 256) return chunk_launch<2, 16>(ctx, a, w, n);
  return chunk_launch<4, 16>(ctx, a, w, n);
}

}  // namespace kanso
