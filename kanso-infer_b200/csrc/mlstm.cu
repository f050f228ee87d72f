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
  const bool four = D % 8 == 0 && V % 8 == 0 && a.width() % 4 == 0 && a.part_stride % 4 == 0;
  auto copy = [&](int64_t from, bf16* to, int n, int ld) {
    if (four) {  // rows without pads: the heads lie one after the other on both sides
      for (int i = threadIdx.x * 4; i < H * n; i += ML_THREADS * 4) {
        float4 v = *reinterpret_cast<const float4*>(a.y + from + i);
        for (int p = 1; p < a.parts; ++p) {
          const float4 u = *reinterpret_cast<const float4*>(a.y + p * a.part_stride + from + i);
          v.x += u.x, v.y += u.y, v.z += u.z, v.w += u.w;
        }
        *reinterpret_cast<uint2*>(to + t * H * ld + i) =
            make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
      }
      return;
    }
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

// A long portion may be cut into segments of whole chunks, which CTAs of their own work on:
//   kCollect  what a segment adds to the state, from nothing, and the sum of its log forget gates
//   (scan)    the state in front of every segment, segment after segment (mlstm_scan_kernel)
//   kEmit     the results of a segment from the state in front of it; the last one leaves the state
// Segments' states lie like slots: segment s of portion p in place p * n + s.
enum MlPass { kWhole, kCollect, kEmit };
struct MlSegments {
  KvStateLayer state;
  uint32_t n = 1, rows = 0;  // segments per portion at most, tokens of one
};

// DW warps along the state's rows (dim), VW along its columns, 16 of them each. A warp's part of
// the transposed state, 16 columns x NT * 8 rows, stays in its registers as accumulators, whose
// layout is that of the A operand which S^T Q^T needs. KB: buffers of keys and values.
constexpr int MC_L = 64, MC_PS = MC_L + 8;

template <int DW, int VW, int NT, int KB>
struct McShape {
  static constexpr int kWarps = DW * VW;
  static constexpr int kThreads = kWarps * 32;
  static constexpr int kCols = VW * 16;         // value columns per CTA
  static constexpr int kDim = DW * NT * 8;      // state rows it can hold
  static constexpr int kQs = kDim + 8, kVs = kCols + 8, kOs = kCols + 4;
  static constexpr size_t kBytes = (size_t)(1 + KB) * MC_L * kQs * 2 + (size_t)KB * MC_L * kVs * 2 +
                                   (size_t)2 * MC_L * MC_PS * 2 + (size_t)kDim * 4 +
                                   (size_t)DW * MC_L * kOs * 4;
};

template <int DW, int VW, int NT, int KB>
__global__ void __launch_bounds__(McShape<DW, VW, NT, KB>::kThreads, 1)
    mlstm_chunk_kernel(const MlstmArgs a, const MlOperands w, const MlSegments seg, MlPass pass) {
  using Sh = McShape<DW, VW, NT, KB>;
  constexpr int QS = Sh::kQs, VS = Sh::kVs, OS = Sh::kOs, COLS = Sh::kCols, NTHR = Sh::kThreads,
                WARPS = Sh::kWarps;
  constexpr int JW = WARPS / 4, NJ = MC_L / JW / 8;  // score columns: groups, tiles of 8 of one
  extern __shared__ __align__(16) uint8_t sm_raw[];
  __shared__ float us[MC_L], gs[MC_L], es[MC_L], as[MC_L], invs[MC_L], dens[JW][MC_L], nqs[MC_L],
      tops[MC_L];
  __shared__ float chunk_m[2];  // G and F at the chunk's end
  bf16* Qs = reinterpret_cast<bf16*>(sm_raw);   // [64][QS]
  bf16* Kb = Qs + MC_L * QS;                    // [KB][64][QS]
  bf16* Vb = Kb + KB * MC_L * QS;               // [KB][64][VS]
  bf16* Ph = Vb + KB * MC_L * VS;               // [64][MC_PS], two parts
  bf16* Pl = Ph + MC_L * MC_PS;
  float* ns = reinterpret_cast<float*>(Pl + MC_L * MC_PS);  // [kDim]
  float* Os = ns + Sh::kDim;                                // [DW][64][OS]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, H = a.heads, D = a.dim, V = a.vdim;
  const int vw = warp / DW, dw = warp % DW;
  const int col0 = blockIdx.x * COLS;           // the CTA's first value column
  const int quad = lane >> 2, two = (lane & 3) * 2;
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t portion = blockIdx.z / seg.n, si = blockIdx.z % seg.n;
  MlPortion p = ml_portion(a, portion);
  bool fresh = p.pos0 == 0, last = true;
  KvStateLayer from = a.state;
  uint32_t from_slot = p.slot;
  if (pass != kWhole) {
    const uint32_t first = si * seg.rows;
    last = first + seg.rows >= p.rows;
    if (first >= p.rows || (pass == kCollect && last)) return;
    p.row0 += first;
    p.rows = min(p.rows - first, seg.rows);
    from = seg.state;
    from_slot = portion * seg.n + si;
    fresh = pass == kCollect;
  }

  // the state: columns vw * 16 + quad (+ 8), rows dw * NT * 8 + nt * 8 + two (+ 1)
  float S[NT][4];
  const int vc = vw * 16 + quad;
  const int tiles = (int)a.state.tiles();
  auto place = [&](const KvStateLayer& l, uint32_t slot, int c, int d) -> float* {
    const int g = col0 + c;
    return l.at(slot, h, g / ML_COLS) + d * ML_COLS + g % ML_COLS;
  };
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = vc + (e >> 1) * 8, d = (dw * NT + nt) * 8 + two + (e & 1);
      S[nt][e] = !fresh && d < D && (col0 + c) / ML_COLS < tiles ? *place(from, from_slot, c, d) : 0.f;
    }
  const float* rec0 = from.at(from_slot, h, col0 / ML_COLS);
  for (int i = tid; i < Sh::kDim; i += NTHR)
    ns[i] = !fresh && i < D ? rec0[a.state.n_at() + i] : 0.f;
  // the sequence starts from a maximum of 0, what a segment adds from none
  float m = pass == kCollect ? -INFINITY
            : fresh          ? 0.f
                             : rec0[a.state.m_at() + (pass == kEmit ? 2 : 0)];
  float f_all = 0.f;

  constexpr int dc = Sh::kDim / 8;
  const int dlc = w.dl / 8, vlc = w.vl / 8;
  auto fetch_qk = [&](const bf16* src, bf16* dst, uint32_t t0) {
    for (int i = tid; i < MC_L * dc; i += NTHR) {
      const int r = i / dc, c = i - r * dc;
      const bool in = t0 + r < p.rows && c < dlc;
      const bf16* at = src + ((p.row0 + (in ? t0 + r : 0)) * H + h) * w.dl + (in ? c : 0) * 8;
      cp_async16(dst + r * QS + c * 8, at, in);
    }
  };
  auto fetch_kv = [&](uint32_t t0, int buf) {
    fetch_qk(w.k, Kb + buf * MC_L * QS, t0);
    for (int i = tid; i < MC_L * (COLS / 8); i += NTHR) {
      const int r = i / (COLS / 8), c = i % (COLS / 8), g = col0 / 8 + c;
      const bool in = t0 + r < p.rows && g < vlc;
      const bf16* at = w.v + ((p.row0 + (in ? t0 + r : 0)) * H + h) * w.vl + (in ? g : 0) * 8;
      cp_async16(Vb + (buf * MC_L + r) * VS + c * 8, at, in);
    }
  };
  if (pass != kCollect) fetch_qk(w.q, Qs, 0);
  fetch_kv(0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  const float scale = 1.0f / sqrtf((float)D);

  int buf = 0;
  for (uint32_t t0 = 0; t0 < p.rows; t0 += MC_L, buf = KB > 1 ? buf ^ 1 : 0) {
    const bool more = t0 + MC_L < p.rows;
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
      tops[lane * 2] = F0 + G0, tops[lane * 2 + 1] = F1 + G1;
      if (lane == 31) {
        chunk_m[0] = G1;
        chunk_m[1] = F1;
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const bf16 *Ks = Kb + buf * MC_L * QS, *Vs = Vb + buf * MC_L * VS;
    if (KB > 1 && more) fetch_kv(t0 + MC_L, buf ^ 1);
    if (KB > 1) asm volatile("cp.async.commit_group;" ::: "memory");
    const uint32_t vt = smem_u32(Vs) + (uint32_t)(((lane & 7) + ((lane >> 4) << 3)) * VS + vw * 16 +
                                                  ((lane >> 3) & 1) * 8) * 2;
    if (pass != kCollect) {
      // n . q, a few tokens per warp
      {
        constexpr int PER = MC_L / WARPS;
        float v[PER];
#pragma unroll
        for (int r = 0; r < PER; ++r) v[r] = 0.f;
        for (int d = lane * 2; d < Sh::kDim; d += 64) {
          const float n0 = ns[d], n1 = ns[d + 1];
#pragma unroll
          for (int r = 0; r < PER; ++r) {
            float x, y;
            unpack_bf16x2(
                *reinterpret_cast<const uint32_t*>(Qs + (warp * PER + r) * QS + d), x, y);
            v[r] = fmaf(x, n0, fmaf(y, n1, v[r]));
          }
        }
#pragma unroll
        for (int r = 0; r < PER; ++r) {
#pragma unroll
          for (int o = 16; o; o >>= 1) v[r] += __shfl_xor_sync(0xFFFFFFFFu, v[r], o);
          if (lane == 0) nqs[warp * PER + r] = v[r] * scale;
        }
      }
      // scores of 16 tokens against NJ * 8, weighted
      {
        const int mt = (warp & 3) * 16, j0 = (warp >> 2) * NJ * 8;
        float c[NJ][4] = {};
        if (j0 <= mt + 15) {
          const uint32_t qa =
              smem_u32(Qs) + (uint32_t)((mt + (lane & 15)) * QS + (lane >> 4) * 8) * 2;
          const uint32_t ka = smem_u32(Ks) +
                              (uint32_t)((j0 + (lane & 7) + ((lane >> 4) << 3)) * QS +
                                         ((lane >> 3) & 1) * 8) * 2;
#pragma unroll 4
          for (int kk = 0; kk < Sh::kDim / 16; ++kk) {
            uint32_t x[4];
            ldm_x4(x, qa + kk * 32);
#pragma unroll
            for (int nt = 0; nt < NJ; nt += 2) {
              uint32_t b[4];
              ldm_x4(b, ka + (uint32_t)(nt * 8 * QS) * 2 + kk * 32);
              mma_bf16(c[nt], x, b[0], b[1]);
              mma_bf16(c[nt + 1], x, b[2], b[3]);
            }
          }
        }
        float sum[2] = {0.f, 0.f};
        const float g0 = gs[mt + quad], g1 = gs[mt + quad + 8];
#pragma unroll
        for (int nt = 0; nt < NJ; ++nt) {
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
      if (more) fetch_qk(w.q, Qs, t0 + MC_L);
      asm volatile("cp.async.commit_group;" ::: "memory");
      if (tid < MC_L) {
        float den = es[tid] * nqs[tid];
#pragma unroll
        for (int k = 0; k < JW; ++k) den += dens[k][tid];
        invs[tid] = 1.0f / (fmaxf(fabsf(den), expf(-tops[tid])) + 1e-6f);
      }
      // the chunk's own tokens: V^T P^T, the keys shared out over the DW warps
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
      float* mine = Os + (size_t)dw * MC_L * OS;
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          mine[(i * 8 + two + (e & 1)) * OS + vc + (e >> 1) * 8] = o[i][e];
    }
    // the state after the chunk
    if (pass != kEmit || more || last) {
      const float GL = chunk_m[0], keep = expf(m - GL);
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
      for (int d = tid; d < Sh::kDim; d += NTHR) {
        float x0 = ns[d] * keep, x1 = 0.f, x2 = 0.f, x3 = 0.f;
#pragma unroll 4
        for (int j = 0; j < MC_L; j += 4) {
          x0 = fmaf(as[j], from_elem(Ks[j * QS + d]), x0);
          x1 = fmaf(as[j + 1], from_elem(Ks[(j + 1) * QS + d]), x1);
          x2 = fmaf(as[j + 2], from_elem(Ks[(j + 2) * QS + d]), x2);
          x3 = fmaf(as[j + 3], from_elem(Ks[(j + 3) * QS + d]), x3);
        }
        ns[d] = x0 + x1 + (x2 + x3);
      }
    }
    f_all += chunk_m[1];
    m = chunk_m[1] + chunk_m[0];
    __syncthreads();  // results are there; keys, values and gates are read out
    if (KB == 1) {
      if (more) fetch_kv(t0 + MC_L, 0);
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
    if (pass != kCollect) {
      for (int i = tid; i < MC_L * COLS; i += NTHR) {
        const int t = i / COLS, c = i % COLS;
        if (t0 + t >= p.rows || col0 + c >= V) continue;
        float v = 0.f;
#pragma unroll
        for (int k = 0; k < DW; ++k) v += Os[(size_t)(k * MC_L + t) * OS + c];
        a.out[(p.row0 + t0 + t) * H * V + (int64_t)h * V + col0 + c] = v * invs[t];
      }
    }
  }
  if (pass == kEmit && !last) return;
  const KvStateLayer to = pass == kCollect ? seg.state : a.state;
  const uint32_t to_slot = pass == kCollect ? from_slot + 1 : p.slot;
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = vc + (e >> 1) * 8, d = (dw * NT + nt) * 8 + two + (e & 1);
      if (d < D && (col0 + c) / ML_COLS < tiles) *place(to, to_slot, c, d) = S[nt][e];
    }
  for (int g = col0 / ML_COLS; g < min(tiles, (col0 + COLS) / ML_COLS); ++g) {
    float* rec = to.at(to_slot, h, g);
    for (int i = tid; i < D; i += NTHR) rec[a.state.n_at() + i] = ns[i];
    if (tid == 0) {
      rec[a.state.m_at()] = m;
      rec[a.state.m_at() + 1] = f_all;  // of use between passes only
    }
  }
}

// The state in front of every segment of a portion, in place of what the segment before it adds;
// blockIdx = (tile and part of its record, head, portion). The maxima in front go to places of
// their own (m_at() + 2): the segments' own are read by other CTAs.
constexpr int MS_PARTS = 4, MS_AHEAD = 4;
__global__ void __launch_bounds__(ML_THREADS) mlstm_scan_kernel(const MlstmArgs a,
                                                               const MlSegments seg) {
  pdl_launch_dependents();
  pdl_wait();
  const MlPortion p = ml_portion(a, blockIdx.z);
  const uint32_t n = (p.rows + seg.rows - 1) / seg.rows, at_m = a.state.m_at();
  const uint32_t tile = blockIdx.x / MS_PARTS, part = blockIdx.x % MS_PARTS;
  const bool fresh = p.pos0 == 0;
  const float* start = a.state.at(p.slot, blockIdx.y, tile);
  const float m0 = fresh ? 0.f : start[at_m];
  const size_t step = seg.state.slot_floats();
  float* base = seg.state.at(blockIdx.z * seg.n, blockIdx.y, tile);
  for (uint32_t i = (part * ML_THREADS + threadIdx.x) * 4; i < at_m;
       i += MS_PARTS * ML_THREADS * 4) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!fresh) v = *reinterpret_cast<const float4*>(start + i);
    *reinterpret_cast<float4*>(base + i) = v;
    float m = m0;
    for (uint32_t s0 = 1; s0 < n; s0 += MS_AHEAD) {
      float4 u[MS_AHEAD];
      float add[MS_AHEAD], f[MS_AHEAD];
#pragma unroll
      for (int k = 0; k < MS_AHEAD; ++k)
        if (s0 + k < n) {
          const float* r = base + (s0 + k) * step;
          u[k] = *reinterpret_cast<const float4*>(r + i);
          add[k] = r[at_m];
          f[k] = r[at_m + 1];
        }
#pragma unroll
      for (int k = 0; k < MS_AHEAD; ++k)
        if (s0 + k < n) {
          const float top = fmaxf(f[k] + m, add[k]);
          const float keep = expf(f[k] + m - top), take = expf(add[k] - top);
          v.x = fmaf(keep, v.x, take * u[k].x), v.y = fmaf(keep, v.y, take * u[k].y);
          v.z = fmaf(keep, v.z, take * u[k].z), v.w = fmaf(keep, v.w, take * u[k].w);
          *reinterpret_cast<float4*>(base + (s0 + k) * step + i) = v;
          m = top;
        }
    }
  }
  if (part == 0 && threadIdx.x == 0) {
    float m = m0;
    base[at_m + 2] = m;
    for (uint32_t s = 1; s < n; ++s) {
      float* r = base + s * step;
      m = fmaxf(r[at_m + 1] + m, r[at_m]);
      r[at_m + 2] = m;
    }
  }
}

template <typename... KArgs, typename... Args>
static int32_t ml_launch(kanso_cuda_ctx* ctx, void (*kern)(KArgs...), dim3 grid, size_t smem,
                         const char* what, int threads, Args... args) {
  int32_t st = allow_max_smem(ctx, (const void*)kern);
  if (st) return st;
  const cudaError_t e = launch_dependent(ctx, kern, grid, dim3(threads), smem, args...);
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
      if (a.dim <= 128) return ml_launch(ctx, mlstm_step_kernel<4>, grid, smem, "mlstm_step", ML_THREADS, a);
      if (a.dim <= 256) return ml_launch(ctx, mlstm_step_kernel<8>, grid, smem, "mlstm_step", ML_THREADS, a);
      return ml_launch(ctx, mlstm_step_kernel<16>, grid, smem, "mlstm_step", ML_THREADS, a);
    }
  }
  const size_t rows = (size_t)3 * ((a.dim + 3) & ~3u) * 4, state = (size_t)a.dim * ML_COLS * 4;
  if (rows > 200 * 1024)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "matrix memory: heads of %u columns", a.dim);
  const int in_smem = rows + state <= 200 * 1024;
  return ml_launch(ctx, mlstm_rows_kernel, grid, rows + (in_smem ? state : 0), "mlstm_rows",
                   ML_THREADS, a, in_smem);
}

bool mlstm_chunk_fits(const MlstmArgs& a) { return a.dim <= 512; }

static size_t ml_room(size_t bytes) { return (bytes + 255) & ~(size_t)255; }
size_t mlstm_chunk_bytes(uint32_t heads, uint32_t dim, uint32_t vdim, int64_t T) {
  const size_t n = (size_t)T * heads;
  return 2 * ml_room(n * round_up8(dim) * 2) + ml_room(n * round_up8(vdim) * 2) +
         2 * ml_room(n * 4);
}

template <int DW, int VW, int NT, int KB>
static int32_t chunk_launch(kanso_cuda_ctx* ctx, const MlstmArgs& a, const MlOperands& w,
                            uint32_t n, uint32_t max_rows) {
  using Sh = McShape<DW, VW, NT, KB>;
  static_assert(Sh::kBytes <= 220 * 1024 && (DW == 2 || DW == 4) && Sh::kCols % ML_COLS == 0, "");
  const unsigned slabs = (a.vdim + Sh::kCols - 1) / Sh::kCols;
  auto kern = mlstm_chunk_kernel<DW, VW, NT, KB>;
  auto pass = [&](const MlSegments& seg, MlPass which) {
    return ml_launch(ctx, kern, dim3(slabs, a.heads, n * seg.n), Sh::kBytes, "mlstm_chunk",
                     Sh::kThreads, a, w, seg, which);
  };
  // as many segments as there are idle SMs for, of two chunks at least
  MlSegments seg;
  const uint32_t chunks = (max_rows + MC_L - 1) / MC_L;
  const uint32_t idle = (uint32_t)std::max(1, ctx->sm_count / (int)(slabs * a.heads * n));
  const uint32_t want = std::min(idle, chunks / 2);
  if (want > 1 && (uint64_t)n * want <= 65535) {
    const uint32_t per = (chunks + want - 1) / want;
    seg.rows = per * MC_L;
    seg.n = (chunks + per - 1) / per;
  }
  if (seg.n == 1) return pass(seg, kWhole);
  seg.state = a.state;
  seg.state.base = (float*)ctx_scratch(ctx, a.state.slot_floats() * n * seg.n * 4);
  if (!seg.state.base) return KANSO_ERR_DEVICE;
  int32_t st = pass(seg, kCollect);
  if (!st)
    st = ml_launch(ctx, mlstm_scan_kernel, dim3(a.state.tiles() * MS_PARTS, a.heads, n), 0, "mlstm_scan",
                   ML_THREADS, a, seg);
  return st ? st : pass(seg, kEmit);
}

int32_t launch_mlstm_chunks(kanso_cuda_ctx* ctx, const MlstmArgs& a, uint32_t n, uint32_t max_rows,
                            void* mem, int64_t T) {
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
  if ((st = ml_launch(ctx, mlstm_operands_kernel, dim3((unsigned)T), 0, "mlstm_operands",
                      ML_THREADS, a, w)))
    return st;
  if (a.dim <= 64) return chunk_launch<2, 4, 4, 2>(ctx, a, w, n, max_rows);
  if (a.dim <= 128) return chunk_launch<4, 4, 4, 2>(ctx, a, w, n, max_rows);
  if (a.dim <= 256) return chunk_launch<4, 4, 8, 2>(ctx, a, w, n, max_rows);
  return chunk_launch<4, 2, 16, 1>(ctx, a, w, n, max_rows);
}

}  // namespace kanso
