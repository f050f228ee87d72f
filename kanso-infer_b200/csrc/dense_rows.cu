// Row-wise pieces of the unquantised models on many rows: scaled embedding, the residual step
// x += mult * rmsnorm(y) * w, the norm of wanted rows, q / k norm with the store to the pool, and
// the routing of rows to experts. All of it in 32-bit; what feeds a matrix product is also
// written in the product's element type.
#include <algorithm>
#include <cmath>

#include "dense.cuh"

namespace kanso {

constexpr int DR_THREADS = 256;

template <typename E>
__global__ void embed_scaled_kernel(const E* __restrict__ embed, int64_t ld,
                                    const uint32_t* __restrict__ tokens, int64_t vocab,
                                    float scale, float* __restrict__ x, int width,
                                    E* __restrict__ xe, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  uint32_t id = tokens[t];
  if (id >= vocab) {
    if (threadIdx.x == 0) atomicOr(status, DEV_BAD_INDEX);
    id = 0;
  }
  for (int i = threadIdx.x; i < ld; i += blockDim.x) {
    const float v = i < width ? from_elem(embed[(int64_t)id * ld + i]) * scale : 0.f;
    if (i < width) x[t * width + i] = v;
    if (xe) xe[t * ld + i] = to_elem<E>(v);
  }
}

__device__ __forceinline__ void add4(float4& a, const float4& b) {
  a.x += b.x, a.y += b.y, a.z += b.z, a.w += b.w;
}
__device__ __forceinline__ float sum_sq4(const float4& v) {
  return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
}
__device__ __forceinline__ void store4(bf16* p, float a, float b, float c, float d) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo),
                                            *reinterpret_cast<const uint32_t*>(&hi));
}
__device__ __forceinline__ void store4(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}

template <typename E>
__global__ void __launch_bounds__(DR_THREADS)
    residual_norm_kernel(float* __restrict__ x, int width, const ResidualSource s,
                         const float* __restrict__ w, float eps, float mult, Residual form,
                         E* __restrict__ xe, int64_t xe_ld) {
  extern __shared__ __align__(16) float v[];  // [width]
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  float* xr = x + t * width;
  const bool after = form == Residual::kAddNorm;  // the norm is of the sum
  const bool four = width % 4 == 0 && s.part_stride % 4 == 0;
  float ss = 0.f;
  if (four) {
#pragma unroll 2
    for (int i = threadIdx.x * 4; i < width; i += DR_THREADS * 4) {
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
      if (s.slot) {
#pragma unroll 4
        for (int j = 0; j < s.top; ++j) {
          const float k = s.weight[t * s.top + j];
          const float4 u = *reinterpret_cast<const float4*>(
              s.y + (int64_t)s.slot[t * s.top + j] * width + i);
          y.x += k * u.x, y.y += k * u.y, y.z += k * u.z, y.w += k * u.w;
        }
      } else {
#pragma unroll 4
        for (int p = 0; p < s.parts; ++p)
          add4(y, *reinterpret_cast<const float4*>(s.y + p * s.part_stride + t * width + i));
      }
      if (after) {
        const float4 r = *reinterpret_cast<const float4*>(xr + i);
        y.x = fmaf(mult, r.x, y.x), y.y = fmaf(mult, r.y, y.y);
        y.z = fmaf(mult, r.z, y.z), y.w = fmaf(mult, r.w, y.w);
      }
      *reinterpret_cast<float4*>(v + i) = y;
      ss += sum_sq4(y);
    }
  } else {
    for (int i = threadIdx.x; i < width; i += DR_THREADS) {
      float y;
      if (s.slot) {
        y = 0.f;
        for (int j = 0; j < s.top; ++j)
          y += s.weight[t * s.top + j] * s.y[(int64_t)s.slot[t * s.top + j] * width + i];
      } else {
        y = s.y[t * width + i];
        for (int p = 1; p < s.parts; ++p) y += s.y[p * s.part_stride + t * width + i];
      }
      if (after) y = fmaf(mult, xr[i], y);
      v[i] = y;
      ss += y * y;
    }
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)width + eps);
  if (four) {
#pragma unroll 2
    for (int i = threadIdx.x * 4; i < width; i += DR_THREADS * 4) {
      const float4 y = *reinterpret_cast<const float4*>(v + i);
      const float4 k = *reinterpret_cast<const float4*>(w + i);
      float4 r;
      if (after) {
        r = make_float4(y.x * inv * k.x, y.y * inv * k.y, y.z * inv * k.z, y.w * inv * k.w);
      } else {
        r = *reinterpret_cast<const float4*>(xr + i);
        r.x += mult * (y.x * inv * k.x), r.y += mult * (y.y * inv * k.y);
        r.z += mult * (y.z * inv * k.z), r.w += mult * (y.w * inv * k.w);
      }
      *reinterpret_cast<float4*>(xr + i) = r;
      if (xe) store4(xe + t * xe_ld + i, r.x, r.y, r.z, r.w);
    }
  } else {
    for (int i = threadIdx.x; i < width; i += DR_THREADS) {
      const float n = v[i] * inv * w[i], r = after ? n : xr[i] + mult * n;
      xr[i] = r;
      if (xe) xe[t * xe_ld + i] = to_elem<E>(r);
    }
  }
  if (xe)
    for (int i = width + threadIdx.x; i < xe_ld; i += DR_THREADS) xe[t * xe_ld + i] = to_elem<E>(0.f);
}

template <typename E>
__global__ void __launch_bounds__(DR_THREADS)
    norm_rows_kernel(const float* __restrict__ x, int width, const uint32_t* __restrict__ rows,
                     const float* __restrict__ w, float eps, E* __restrict__ out, int64_t out_ld) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const float* xr = x + (int64_t)(rows ? rows[blockIdx.x] : blockIdx.x) * width;
  E* o = out + (int64_t)blockIdx.x * out_ld;
  float ss = 0.f;
  for (int i = threadIdx.x; i < width; i += DR_THREADS) ss += xr[i] * xr[i];
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)width + eps);
  for (int i = threadIdx.x; i < out_ld; i += DR_THREADS)
    o[i] = to_elem<E>(i < width ? xr[i] * inv * w[i] : 0.f);
}

template <typename E>
__global__ void __launch_bounds__(DR_THREADS)
    qk_norm_store_kernel(const QkvSource s, const KvDenseLayer kv, int H, const RowMap map,
                         E* __restrict__ q_out, int* status) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const int D = kv.k_dim, DV = kv.v_dim, G = kv.kv_heads;
  const int nq = H * D, nk = G * D, nv = G * DV;
  const int64_t width = nq + nk + nv;
  const float* src = s.qkv + t * width;
  auto value = [&](int i) {
    float v = src[i];
    for (int p = 1; p < s.parts; ++p) v += src[p * s.part_stride + i];
    return v;
  };
  const uint32_t pos = map.positions[t];
  const uint32_t seq = map.row_seq ? map.row_seq[t] : (uint32_t)t;
  const uint32_t place = pos / kv.block_size, off = pos % kv.block_size;
  uint32_t block = kv.num_blocks;
  if (place < map.max_blocks) block = map.tables[(int64_t)seq * map.max_blocks + place];
  const bool ok = block < kv.num_blocks;
  if (!ok && threadIdx.x == 0) atomicOr(status, DEV_BAD_INDEX);
  E* pool = reinterpret_cast<E*>(kv.base);

  if (D % 8 == 0 && DV % 8 == 0 && s.part_stride % 4 == 0) {
    // rows without pads, four columns at a time; the sums of the parts stay in shared memory
    extern __shared__ __align__(16) float row[];  // [width]
    float sq = 0.f, sk = 0.f;
#pragma unroll 4
    for (int i = threadIdx.x * 4; i < (int)width; i += DR_THREADS * 4) {
      float4 v = *reinterpret_cast<const float4*>(src + i);
      for (int p = 1; p < s.parts; ++p)
        add4(v, *reinterpret_cast<const float4*>(src + p * s.part_stride + i));
      *reinterpret_cast<float4*>(row + i) = v;
      if (i < nq)
        sq += sum_sq4(v);
      else if (i < nq + nk)
        sk += sum_sq4(v);
    }
    sq = block_sum(sq, red);
    sk = block_sum(sk, red);
    const float iq = 1.0f / sqrtf(sq / (float)nq + s.eps), ik = 1.0f / sqrtf(sk / (float)nk + s.eps);
    for (int i = threadIdx.x * 4; i < (int)width; i += DR_THREADS * 4) {
      float4 v = *reinterpret_cast<const float4*>(row + i);
      if (i < nq + nk) {
        const float f = i < nq ? iq : ik;
        const float4 n = *reinterpret_cast<const float4*>(i < nq ? s.q_norm + i : s.k_norm + i - nq);
        v.x *= f * n.x, v.y *= f * n.y, v.z *= f * n.z, v.w *= f * n.w;
      }
      E* dst = q_out + t * nq + i;
      if (i >= nq + nk) {
        const int c = i - nq - nk, g = c / DV;
        dst = pool + kv.v_elem(ok ? block : 0u, g, off) + (c - g * DV);
      } else if (i >= nq) {
        const int c = i - nq, g = c / D;
        dst = pool + kv.k_elem(ok ? block : 0u, g, off) + (c - g * D);
      }
      if (ok || i < nq) store4(dst, v.x, v.y, v.z, v.w);
    }
    return;
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < nq; i += DR_THREADS) {
    const float v = value(i);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  float inv = 1.0f / sqrtf(ss / (float)nq + s.eps);
  for (int i = threadIdx.x; i < H * (int)kv.k_ld; i += DR_THREADS) {
    const int h = i / kv.k_ld, d = i - h * kv.k_ld;
    const float v = d < D ? value(h * D + d) * inv * s.q_norm[h * D + d] : 0.f;
    q_out[t * H * kv.k_ld + i] = to_elem<E>(v);
  }
  ss = 0.f;
  for (int i = threadIdx.x; i < nk; i += DR_THREADS) {
    const float v = value(nq + i);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  if (!ok) return;
  inv = 1.0f / sqrtf(ss / (float)nk + s.eps);
  for (int i = threadIdx.x; i < G * (int)kv.k_ld; i += DR_THREADS) {
    const int g = i / kv.k_ld, d = i - g * kv.k_ld;
    const float v = d < D ? value(nq + g * D + d) * inv * s.k_norm[g * D + d] : 0.f;
    pool[kv.k_elem(block, g, off) + d] = to_elem<E>(v);
  }
  for (int i = threadIdx.x; i < G * (int)kv.v_ld; i += DR_THREADS) {
    const int g = i / kv.v_ld, d = i - g * kv.v_ld;
    const float v = d < DV ? value(nq + nk + g * DV + d) : 0.f;
    pool[kv.v_elem(block, g, off) + d] = to_elem<E>(v);
  }
}

__global__ void expert_sum_kernel(const float* __restrict__ ye, const uint32_t* __restrict__ slot,
                                  const float* __restrict__ weight, int top, float* __restrict__ y,
                                  int width) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float v = 0.f;
    for (int j = 0; j < top; ++j)
      v += weight[t * top + j] * ye[(int64_t)slot[t * top + j] * width + i];
    y[t * width + i] = v;
  }
}

// Router and choice, one CTA per RW rows: its warps share out the experts, two at a time
// (logits = router . x + bias in f32), then one warp per row makes the choice (warp_route).
template <int RW>
__global__ void __launch_bounds__(DR_THREADS)
    route_kernel(const float* __restrict__ x, int width, const float* __restrict__ router, int ld,
                 const float* __restrict__ bias, int experts, int top, RouteWeights form, uint32_t* __restrict__ sel, float* __restrict__ weight,
                 uint32_t* __restrict__ counts, uint32_t* __restrict__ slot, int64_t T) {
  extern __shared__ __align__(16) float sm[];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t t0 = (int64_t)blockIdx.x * RW;
  float* xw = sm;             // [RW][ld]
  float* l = xw + RW * ld;    // [RW][experts]
#pragma unroll
  for (int r = 0; r < RW; ++r)
    for (int i = threadIdx.x; i < ld; i += DR_THREADS)
      xw[r * ld + i] = i < width && t0 + r < T ? x[(t0 + r) * width + i] : 0.f;
  __syncthreads();
  for (int e0 = warp * 2; e0 < experts; e0 += DR_THREADS / 32 * 2) {
    const float* w0 = router + (int64_t)e0 * ld;
    const float* w1 = router + (int64_t)min(e0 + 1, experts - 1) * ld;
    float acc[RW * 2];
#pragma unroll
    for (int i = 0; i < RW * 2; ++i) acc[i] = 0.f;
#pragma unroll 4
    for (int c = lane * 4; c < ld; c += 128) {
      const float4 a = *reinterpret_cast<const float4*>(w0 + c);
      const float4 b = *reinterpret_cast<const float4*>(w1 + c);
#pragma unroll
      for (int r = 0; r < RW; ++r) {
        const float4 v = *reinterpret_cast<const float4*>(xw + r * ld + c);
        float s = acc[r * 2], u = acc[r * 2 + 1];
        s = fmaf(a.x, v.x, s), u = fmaf(b.x, v.x, u);
        s = fmaf(a.y, v.y, s), u = fmaf(b.y, v.y, u);
        s = fmaf(a.z, v.z, s), u = fmaf(b.z, v.z, u);
        acc[r * 2] = fmaf(a.w, v.w, s), acc[r * 2 + 1] = fmaf(b.w, v.w, u);
      }
    }
#pragma unroll
    for (int i = 0; i < RW * 2; ++i) {
#pragma unroll
      for (int o = 16; o; o >>= 1) acc[i] += __shfl_xor_sync(0xFFFFFFFFu, acc[i], o);
      const int e = e0 + i % 2;
      if (lane == 0 && e < experts) l[i / 2 * experts + e] = acc[i] + (bias ? bias[e] : 0.f);
    }
  }
  __syncthreads();
  const int64_t t = t0 + warp;
  if (warp >= RW || t >= T) return;
  warp_route(l + warp * experts, experts, top, form, lane, sel + t * top, weight + t * top);
  for (int j = lane; j < top; j += 32)
    slot[t * top + j] = atomicAdd(&counts[sel[t * top + j]], 1u);
}

// Every CTA forms the offsets from the counts (one warp, a running scan) and moves its rows.
template <typename E>
__global__ void __launch_bounds__(DR_THREADS)
    expert_gather_kernel(const uint32_t* __restrict__ counts, int experts, int top,
                         const uint32_t* __restrict__ sel, uint32_t* __restrict__ slot,
                         uint32_t* __restrict__ offsets, const E* __restrict__ xe, int64_t ld,
                         E* __restrict__ xs) {
  extern __shared__ uint32_t off[];  // [experts + 1]
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  if (threadIdx.x < 32) {
    uint32_t carry = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const uint32_t n = e < experts ? counts[e] : 0u;
      uint32_t incl = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const uint32_t v = __shfl_up_sync(0xFFFFFFFFu, incl, o);
        if ((int)threadIdx.x >= o) incl += v;
      }
      if (e < experts) off[e] = carry + incl - n;
      carry += __shfl_sync(0xFFFFFFFFu, incl, 31);
    }
    if (threadIdx.x == 0) off[experts] = carry;
  }
  __syncthreads();
  if (t == 0)
    for (int e = threadIdx.x; e <= experts; e += DR_THREADS) offsets[e] = off[e];
  const int vec = (int)(ld * sizeof(E) / 16);
  const uint4* src = reinterpret_cast<const uint4*>(xe + t * ld);
  for (int j = 0; j < top; ++j) {
    const uint32_t row = off[sel[t * top + j]] + slot[t * top + j];
    uint4* dst = reinterpret_cast<uint4*>(xs + (int64_t)row * ld);
    for (int i = threadIdx.x; i < vec; i += DR_THREADS) dst[i] = src[i];
  }
  __syncthreads();  // every thread has read the places before they become rows
  for (int j = threadIdx.x; j < top; j += DR_THREADS) slot[t * top + j] += off[sel[t * top + j]];
}

// ---- latent attention: what happens to its rows around the products ----
template <typename E>
__global__ void __launch_bounds__(DR_THREADS)
    latent_down_kernel(const LatentStore s, E* __restrict__ cq, int64_t cq_ld) {
  __shared__ float red[32];
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  if (blockIdx.y == 1) {  // the cache row
    const float2 turn = latent_turn(s, t);
    pdl_wait();
    latent_store_row<E>(s, t, turn, red);
    return;
  }
  pdl_wait();
  const LatentDown& p = s.down;
  const float* src = p.d + t * p.ld;
  const int Q = (int)p.q_rank;
  auto value = [&](int i) {
    float v = src[i];
#pragma unroll 3
    for (int k = 1; k < p.parts; ++k) v += src[k * p.part_stride + i];
    return v;
  };
  constexpr int KEEP = 6;  // values a thread keeps between the two passes
  float kept[KEEP], ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = threadIdx.x + k * DR_THREADS;
    kept[k] = i < Q ? value(i) : 0.f;
    ss += kept[k] * kept[k];
  }
  for (int i = threadIdx.x + KEEP * DR_THREADS; i < Q; i += DR_THREADS) {
    const float v = value(i);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)Q + p.eps);
  E* dst = cq + t * cq_ld;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = threadIdx.x + k * DR_THREADS;
    if (i < cq_ld) dst[i] = to_elem<E>(i < Q ? kept[k] * inv * p.q_norm[i] : 0.f);
  }
  for (int i = threadIdx.x + KEEP * DR_THREADS; i < cq_ld; i += DR_THREADS)
    dst[i] = to_elem<E>(i < Q ? value(i) * inv * p.q_norm[i] : 0.f);
}

// blockIdx.y = a part of the heads
template <typename E>
__global__ void __launch_bounds__(DR_THREADS)
    latent_q_heads_kernel(const LatentAttn a, const LatentQuery q, const uint32_t* __restrict__ rows,
                          int64_t n, E* __restrict__ out, int ld) {
  pdl_launch_dependents();
  const int64_t i = blockIdx.x, t = rows ? rows[i] : i;
  const int per = ((int)a.heads + gridDim.y - 1) / gridDim.y, h0 = blockIdx.y * per,
            h1 = min(h0 + per, (int)a.heads), D = a.dim, Q = D + a.rot;
  const float* src = q.q + t * q.ld;
  pdl_wait();
  if (D % 8 == 0 && Q % 4 == 0 && q.ld % 4 == 0 && q.part_stride % 4 == 0) {
    for (int k = threadIdx.x * 4; k < (h1 - h0) * D; k += DR_THREADS * 4) {
      const int h = h0 + k / D, d = k % D;
      const float* at = src + (int64_t)h * Q + d;
      float4 v = *reinterpret_cast<const float4*>(at);
#pragma unroll 3
      for (int p = 1; p < q.parts; ++p)
        add4(v, *reinterpret_cast<const float4*>(at + p * q.part_stride));
      store4(out + ((int64_t)h * n + i) * ld + d, v.x, v.y, v.z, v.w);
    }
    return;
  }
  for (int k = threadIdx.x; k < (h1 - h0) * ld; k += DR_THREADS) {
    const int h = h0 + k / ld, d = k % ld;
    float v = 0.f;
    if (d < D) {
      const float* at = src + (int64_t)h * Q + d;
      v = at[0];
      for (int p = 1; p < q.parts; ++p) v += at[p * q.part_stride];
    }
    out[((int64_t)h * n + i) * ld + d] = to_elem<E>(v);
  }
}

__global__ void __launch_bounds__(DR_THREADS)
    latent_q_rows_kernel(const LatentAttn a, const LatentQuery q,
                         const uint32_t* __restrict__ positions, bf16* __restrict__ out, int ld,
                         bf16* __restrict__ out_rot, int rot_ld) {
  extern __shared__ float2 turn[];  // [rot / 2] (sin, cos)
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  for (int i = threadIdx.x; i < (int)a.rot / 2; i += DR_THREADS)
    rope_sincos(positions[t], a.freq[i], &turn[i].x, &turn[i].y);
  pdl_wait();
  __syncthreads();
  const float* src = q.q + t * q.ld;
  const int D = a.dim, RD = a.rot, H = a.heads;
  auto value = [&](int64_t i) {
    float v = src[i];
    for (int p = 1; p < q.parts; ++p) v += src[p * q.part_stride + i];
    return v;
  };
  // two columns at a time (the leading dimensions are even)
  for (int k = threadIdx.x * 2; k < H * ld; k += DR_THREADS * 2) {
    const int h = k / ld, d = k - h * ld;
    const int64_t at = (int64_t)h * (D + RD) + d;
    const float u = d < D ? value(at) : 0.f, v = d + 1 < D ? value(at + 1) : 0.f;
    *reinterpret_cast<__nv_bfloat162*>(out + (t * H + h) * ld + d) = __floats2bfloat162_rn(u, v);
  }
  for (int k = threadIdx.x * 2; k < H * rot_ld; k += DR_THREADS * 2) {
    const int h = k / rot_ld, d = k - h * rot_ld;
    float u = 0.f, v = 0.f;
    if (d < RD) {
      const int64_t at = (int64_t)h * (D + RD) + D + d;
      const float x = value(at), y = value(at + 1);
      const float2 sc = turn[d / 2];
      u = x * sc.y - y * sc.x;
      v = y * sc.y + x * sc.x;
    }
    *reinterpret_cast<__nv_bfloat162*>(out_rot + (t * H + h) * rot_ld + d) =
        __floats2bfloat162_rn(u, v);
  }
}

// A warp per cache row.
__global__ void __launch_bounds__(DR_THREADS)
    latent_gather_kernel(const KvDenseLayer kv, const RowMap map, const AttnTile* __restrict__ runs,
                         int n_runs, int R, int RD, bf16* __restrict__ c, int c_ld,
                         bf16* __restrict__ rot, int rot_ld, int64_t n, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = ((int64_t)blockIdx.x * DR_THREADS + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (i >= n) return;
  int r = 0;
  while (r + 1 < n_runs && i >= runs[r + 1].row0) ++r;
  const uint32_t j = (uint32_t)(i - runs[r].row0), seq = runs[r].pos0, place = j / kv.block_size;
  uint32_t block = kv.num_blocks;
  if (place < map.max_blocks) block = map.tables[(int64_t)seq * map.max_blocks + place];
  if (block >= kv.num_blocks) {
    if (lane == 0) atomicOr(status, DEV_BAD_INDEX);
    block = 0;
  }
  const bf16* src = reinterpret_cast<const bf16*>(kv.base) + kv.k_elem(block, 0, j % kv.block_size);
  if (R % 8 == 0) {
    for (int d = lane * 8; d < R; d += 256)
      *reinterpret_cast<uint4*>(c + i * c_ld + d) = *reinterpret_cast<const uint4*>(src + d);
  } else {
    for (int d = lane; d < c_ld; d += 32) c[i * c_ld + d] = d < R ? src[d] : to_elem<bf16>(0.f);
  }
  for (int d = lane; d < rot_ld; d += 32)
    rot[i * rot_ld + d] = d < RD ? src[R + d] : to_elem<bf16>(0.f);
}

// ---- matrix memory: the heads' outputs on the way to the o-projection ----
// One CTA per head and row.
constexpr int HN_THREADS = 128;
template <typename E>
__global__ void __launch_bounds__(HN_THREADS)
    head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ gate,
                          int64_t gate_ld, int parts, int64_t part_stride, int heads, int hd,
                          const float* __restrict__ w, float eps, E* __restrict__ out,
                          int64_t out_ld) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, n = heads * hd;
  const int64_t t = blockIdx.y;
  const float *x = o + t * n + h * hd, *g = gate + t * gate_ld + h * hd;
  E* dst = out + t * out_ld + h * hd;
  w += h * hd;
  float ss = 0.f;
  if (hd % 4 == 0 && gate_ld % 4 == 0 && part_stride % 4 == 0 &&
      ((reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) & 15u) == 0 &&
      out_ld % 4 == 0) {
    for (int i = threadIdx.x * 4; i < hd; i += HN_THREADS * 4)
      ss += sum_sq4(*reinterpret_cast<const float4*>(x + i));
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)hd + eps);
    for (int i = threadIdx.x * 4; i < hd; i += HN_THREADS * 4) {
      const float4 v = *reinterpret_cast<const float4*>(x + i);
      const float4 k = *reinterpret_cast<const float4*>(w + i);
      float4 z = *reinterpret_cast<const float4*>(g + i);
#pragma unroll 3
      for (int p = 1; p < parts; ++p)
        add4(z, *reinterpret_cast<const float4*>(g + p * part_stride + i));
      store4(dst + i, v.x * inv * k.x / (1.0f + expf(-z.x)), v.y * inv * k.y / (1.0f + expf(-z.y)),
             v.z * inv * k.z / (1.0f + expf(-z.z)), v.w * inv * k.w / (1.0f + expf(-z.w)));
    }
  } else {
    for (int i = threadIdx.x; i < hd; i += HN_THREADS) ss += x[i] * x[i];
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)hd + eps);
    for (int i = threadIdx.x; i < hd; i += HN_THREADS) {
      float z = g[i];
      for (int p = 1; p < parts; ++p) z += g[p * part_stride + i];
      dst[i] = to_elem<E>(x[i] * inv * w[i] / (1.0f + expf(-z)));
    }
  }
  if (h == heads - 1)
    for (int i = n + threadIdx.x; i < out_ld; i += HN_THREADS) out[t * out_ld + i] = to_elem<E>(0.f);
}

#define DR_LAUNCH(kern, grid, threads, smem, what, ...)                                          \
  do {                                                                                           \
    const cudaError_t e_ = launch_dependent(ctx, kern, dim3((unsigned)(grid)), dim3(threads),    \
                                            smem, __VA_ARGS__);                                  \
    if (e_ != cudaSuccess) return cuda_fail(ctx, e_, what);                                      \
    return after_launch(ctx, what);                                                              \
  } while (0)

int32_t launch_embed_scaled(kanso_cuda_ctx* ctx, int32_t compute, const void* embed, int64_t ld,
                            const uint32_t* tokens, int64_t vocab, float scale, float* x,
                            int64_t width, void* xe, int64_t T) {
  // a plain launch: a step's first kernel starts when everything before the step has ended
  if (compute == KANSO_COMPUTE_BF16)
    embed_scaled_kernel<bf16><<<(unsigned)T, DR_THREADS, 0, ctx->stream>>>(
        (const bf16*)embed, ld, tokens, vocab, scale, x, (int)width, (bf16*)xe, ctx->dev_status);
  else
    embed_scaled_kernel<float><<<(unsigned)T, DR_THREADS, 0, ctx->stream>>>(
        (const float*)embed, ld, tokens, vocab, scale, x, (int)width, (float*)xe, ctx->dev_status);
  return after_launch(ctx, "embed_scaled");
}

int32_t launch_residual_norm(kanso_cuda_ctx* ctx, int32_t compute, float* x, int64_t width,
                             const ResidualSource& s, const float* w, float eps, float mult,
                             Residual form, void* xe, int64_t xe_ld, int64_t T) {
  const size_t smem = (size_t)width * 4;
  if (smem > 200 * 1024)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "residual norm: width %lld", (long long)width);
  auto kern_b = residual_norm_kernel<bf16>;
  auto kern_f = residual_norm_kernel<float>;
  int32_t st = allow_max_smem(ctx, compute == KANSO_COMPUTE_BF16 ? (const void*)kern_b
                                                                 : (const void*)kern_f);
  if (st) return st;
  if (compute == KANSO_COMPUTE_BF16)
    DR_LAUNCH(kern_b, T, DR_THREADS, smem, "residual_norm", x, (int)width, s, w, eps, mult,
              form, (bf16*)xe, xe_ld);
  DR_LAUNCH(kern_f, T, DR_THREADS, smem, "residual_norm", x, (int)width, s, w, eps, mult,
            form, (float*)xe, xe_ld);
}

int32_t launch_expert_sum(kanso_cuda_ctx* ctx, const float* ye, const uint32_t* slot,
                          const float* weight, uint32_t top, float* y, int64_t width, int64_t T) {
  DR_LAUNCH(expert_sum_kernel, T, DR_THREADS, 0, "expert_sum", ye, slot, weight, (int)top, y,
            (int)width);
}

int32_t launch_norm_rows(kanso_cuda_ctx* ctx, int32_t compute, const float* x, int64_t width,
                         const uint32_t* rows, const float* w, float eps, void* out,
                         int64_t out_ld, int64_t n) {
  if (compute == KANSO_COMPUTE_BF16)
    DR_LAUNCH(norm_rows_kernel<bf16>, n, DR_THREADS, 0, "norm_rows", x, (int)width, rows, w, eps,
              (bf16*)out, out_ld);
  DR_LAUNCH(norm_rows_kernel<float>, n, DR_THREADS, 0, "norm_rows", x, (int)width, rows, w, eps,
            (float*)out, out_ld);
}

int32_t launch_qk_norm_store(kanso_cuda_ctx* ctx, int32_t compute, const QkvSource& s,
                             const KvDenseLayer& kv, uint32_t H, const RowMap& map, void* q_out,
                             int64_t T) {
  const size_t width = (size_t)H * kv.k_dim + (size_t)kv.kv_heads * (kv.k_dim + kv.v_dim);
  const bool vec = kv.k_dim % 8 == 0 && kv.v_dim % 8 == 0 && s.part_stride % 4 == 0;
  const size_t smem = vec ? width * 4 : 0;
  if (smem > 200 * 1024)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "qk norm: %zu columns of q, k and v", width);
  auto kern_b = qk_norm_store_kernel<bf16>;
  auto kern_f = qk_norm_store_kernel<float>;
  int32_t st = allow_max_smem(ctx, compute == KANSO_COMPUTE_BF16 ? (const void*)kern_b
                                                                 : (const void*)kern_f);
  if (st) return st;
  if (compute == KANSO_COMPUTE_BF16)
    DR_LAUNCH(kern_b, T, DR_THREADS, smem, "qk_norm_store", s, kv, (int)H, map, (bf16*)q_out,
              ctx->dev_status);
  DR_LAUNCH(kern_f, T, DR_THREADS, smem, "qk_norm_store", s, kv, (int)H, map, (float*)q_out,
            ctx->dev_status);
}

int32_t launch_route(kanso_cuda_ctx* ctx, const float* x, int64_t width, const DenseMat& router,
                     const float* bias, uint32_t top, RouteWeights form, uint32_t* sel, float* weight, uint32_t* counts, uint32_t* slot,
                     int64_t T) {
  const int experts = (int)router.rows, ld = (int)router.ld;
  // four rows per CTA where that leaves every SM two of them
  const int rw = T >= 8 * (int64_t)ctx->sm_count && ld <= 8192 ? 4 : 1;
  const size_t smem = (size_t)rw * (ld + experts) * 4;
  if (smem > 220 * 1024)
    return fail(ctx, KANSO_ERR_UNSUPPORTED, "router: %d experts, width %lld", experts,
                (long long)width);
  auto kern = rw == 4 ? route_kernel<4> : route_kernel<1>;
  int32_t st = allow_max_smem(ctx, (const void*)kern);
  if (st) return st;
  DR_LAUNCH(kern, (T + rw - 1) / rw, DR_THREADS, smem, "route", x, (int)width,
            (const float*)router.w, ld, bias, experts, (int)top, form, sel, weight, counts, slot, T);
}

int32_t launch_expert_gather(kanso_cuda_ctx* ctx, int32_t compute, const uint32_t* counts,
                             uint32_t experts, uint32_t top, const uint32_t* sel, uint32_t* slot,
                             uint32_t* offsets, const void* xe, int64_t ld, void* xs, int64_t T) {
  const size_t smem = ((size_t)experts + 1) * 4;
  if (compute == KANSO_COMPUTE_BF16)
    DR_LAUNCH(expert_gather_kernel<bf16>, T, DR_THREADS, smem, "expert_gather", counts,
              (int)experts, (int)top, sel, slot, offsets, (const bf16*)xe, ld, (bf16*)xs);
  DR_LAUNCH(expert_gather_kernel<float>, T, DR_THREADS, smem, "expert_gather", counts,
            (int)experts, (int)top, sel, slot, offsets, (const float*)xe, ld, (float*)xs);
}

std::vector<double> rope_frequencies(uint32_t dims, double base) {
  std::vector<double> f(dims / 2);
  for (uint32_t i = 0; i < dims / 2; ++i) f[i] = std::pow(base, -2.0 * i / dims);
  return f;
}

int32_t launch_latent_down(kanso_cuda_ctx* ctx, int32_t compute, const LatentStore& s, void* cq,
                           int64_t T) {
  const int64_t ld = round_up8(s.down.q_rank);
  const dim3 grid((unsigned)T, 2);
  const cudaError_t e =
      compute == KANSO_COMPUTE_BF16
          ? launch_dependent(ctx, latent_down_kernel<bf16>, grid, dim3(DR_THREADS), 0, s, (bf16*)cq,
                             ld)
          : launch_dependent(ctx, latent_down_kernel<float>, grid, dim3(DR_THREADS), 0, s,
                             (float*)cq, ld);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "latent_down");
  return after_launch(ctx, "latent_down");
}

int32_t launch_latent_q_heads(kanso_cuda_ctx* ctx, int32_t compute, const LatentAttn& a,
                              const LatentQuery& q, const uint32_t* rows, int64_t n, void* out) {
  const int ld = (int)round_up8(a.dim);
  // few rows: a thread's four columns in one go
  const int64_t trips = ((int64_t)a.heads * ld + DR_THREADS * 4 - 1) / (DR_THREADS * 4);
  const dim3 grid((unsigned)n, (unsigned)std::min<int64_t>({trips, (int64_t)a.heads, n > 512 ? 1 : 8}));
  const cudaError_t e =
      compute == KANSO_COMPUTE_BF16
          ? launch_dependent(ctx, latent_q_heads_kernel<bf16>, grid, dim3(DR_THREADS), 0, a, q,
                             rows, n, (bf16*)out, ld)
          : launch_dependent(ctx, latent_q_heads_kernel<float>, grid, dim3(DR_THREADS), 0, a, q,
                             rows, n, (float*)out, ld);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "latent_q_heads");
  return after_launch(ctx, "latent_q_heads");
}

int32_t launch_latent_q_rows(kanso_cuda_ctx* ctx, const LatentAttn& a, const LatentQuery& q,
                             const uint32_t* positions, bf16* out, bf16* out_rot, int64_t T) {
  DR_LAUNCH(latent_q_rows_kernel, T, DR_THREADS, (size_t)a.rot * 4, "latent_q_rows", a, q, positions,
            out, (int)round_up8(a.dim), out_rot, (int)round_up8(a.rot));
}

int32_t launch_latent_gather(kanso_cuda_ctx* ctx, const LatentAttn& a, const KvDenseLayer& kv,
                             const RowMap& map, const AttnTile* runs, uint32_t n_runs, bf16* c,
                             bf16* rot, int64_t n) {
  DR_LAUNCH(latent_gather_kernel, (n + DR_THREADS / 32 - 1) / (DR_THREADS / 32), DR_THREADS, 0,
            "latent_gather", kv, map, runs, (int)n_runs, (int)a.rank, (int)a.rot, c,
            (int)round_up8(a.rank), rot, (int)round_up8(a.rot), n, ctx->dev_status);
}

int32_t launch_head_norm_gate(kanso_cuda_ctx* ctx, int32_t compute, const MlstmArgs& a,
                              const float* w, float eps, void* out, int64_t out_ld, int64_t T) {
  const int H = a.heads, V = a.vdim;
  const float* gate = a.y + (int64_t)H * (2 * a.dim + V);
  const dim3 grid((unsigned)H, (unsigned)T);
  const cudaError_t e =
      compute == KANSO_COMPUTE_BF16
          ? launch_dependent(ctx, head_norm_gate_kernel<bf16>, grid, dim3(HN_THREADS), 0, a.out,
                             gate, a.width(), a.parts, a.part_stride, H, V, w, eps, (bf16*)out,
                             out_ld)
          : launch_dependent(ctx, head_norm_gate_kernel<float>, grid, dim3(HN_THREADS), 0, a.out,
                             gate, a.width(), a.parts, a.part_stride, H, V, w, eps, (float*)out,
                             out_ld);
  if (e != cudaSuccess) return cuda_fail(ctx, e, "head_norm_gate");
  return after_launch(ctx, "head_norm_gate");
}

}  // namespace kanso
