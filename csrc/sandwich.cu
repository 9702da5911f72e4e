// Sandwich-norm hybrid decoders (Nipudra) -- what the fused projections, the paged softmax attention and the linear recurrences
// of seqmix.cu do not have yet:
//   * sandwich_join    x <- x + N_b(y), h = N_a(x): the norm behind a sublayer, the residual addition and the norm in front of the
//                      next sublayer in one pass; either norm is a layer norm (weight and bias) or an RMS norm, h may also be a
//                      plain copy of the residual as the operand of a matrix product
//   * rot_table        cos and sin of every rotary pair of every token of a step, once per distinct set of frequencies
//   * conv_rot_prep    short causal convolutions on q, k and v, rotary positions (pairs i, i + half), K / V rows into the cache
//   * rot_cast         rotary positions (pairs 2i, 2i + 1) on q and k of a recurrence, bf16 rows of q, k and v
//   * diff_combine     differential attention: a_1 - lambda a_2 of a head's two maps, divided by its root mean square
//   * ssd_post         (recurrence output + D x) * silu(z), RMS norm in equal parts, weight -> operand
//   * side_gate        gelu(z) * the token's own channels for this layer -> operand
// Norms, angles and the residual are fp32 in every mode; OT / CT (operand / cache type) is bf16 or float.
// This translation unit is compiled WITHOUT --use_fast_math (exact expf / tanhf / division / sqrt / sincos).
#include "kernels.h"

#include <cuda_bf16.h>

#include <cstdint>

#include "launch.cuh"

namespace b2b {
namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ void stf(float* p, size_t i, float v) { p[i] = v; }
__device__ __forceinline__ void stf(bf16* p, size_t i, float v) { p[i] = __float2bfloat16_rn(v); }
__device__ __forceinline__ float ldf(const float* p, size_t i) { return p[i]; }
__device__ __forceinline__ float ldf(const bf16* p, size_t i) { return __bfloat162float(p[i]); }
__device__ __forceinline__ void st4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(bf16* p, const float4& v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<unsigned*>(&a);
  u.y = *reinterpret_cast<unsigned*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

__device__ __forceinline__ void pdl_begin() {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
}
__device__ __forceinline__ float warp_sum_(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// sum over the block; every thread gets the result (sh: >= 32 floats, reusable after the call)
__device__ __forceinline__ float block_sum_(float v, float* sh) {
  v = warp_sum_(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (nw == 1) return v;
  __syncthreads();
  if (l == 0) sh[w] = v;
  __syncthreads();
  return warp_sum_(l < nw ? sh[l] : 0.f);
}
__device__ __forceinline__ float silu_(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float gelu_tanh_(float z) {
  return 0.5f * z * (1.f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
}
// sin and cos of position * (fhi + flo): the fp32 product pos * fhi is corrected by what its rounding lost and by pos * flo
// through the addition formulas, so far positions keep the last bits of the angle
__device__ __forceinline__ void turn_(float pos, float fhi, float flo, float* sn, float* cs) {
  const float a = __fmul_rn(pos, fhi);
  const float r = __fmaf_rn(pos, flo, __fmaf_rn(pos, fhi, -a));
  float s, c, sr, cr;
  sincosf(a, &s, &c);
  sincosf(r, &sr, &cr);
  *sn = __fmaf_rn(s, cr, c * sr);
  *cs = __fmaf_rn(c, cr, -s * sr);
}

// ------------------------------------------------------------------------------------------- join between two norms
// One block per row.  rows == nullptr: row = token, x is updated in place; rows != nullptr: row r reads token rows[r] and only
// h[r] is written.  y (optional, indexed by token): x += N_y(y).  Norm kinds: 0 root mean square with a weight, 1 layer norm
// (mean taken off; the variance is the mean of the squared deviations) with weight and bias, 2 (h only) none.
// VEC: 16-byte accesses; NV vectors (or single values) per thread stay in registers.
enum { NORM_RMS = 0, NORM_LAYER = 1, NORM_NONE = 2 };

template <int E, int NV>
__device__ __forceinline__ void row_stats(const float (&v)[NV][E], int nv, int W, int kind, float eps, float* red, float* mean,
                                          float* rinv) {
  float m = 0.f;
  if (kind == NORM_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k)
#pragma unroll
      for (int e = 0; e < E; ++e) s += v[k][e];             // (elements behind the row are zero)
    m = block_sum_(s, red) / static_cast<float>(W);
  }
  float q = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    if (k * static_cast<int>(blockDim.x) + static_cast<int>(threadIdx.x) < nv) {
#pragma unroll
      for (int e = 0; e < E; ++e) {
        const float d = v[k][e] - m;
        q += d * d;
      }
    }
  }
  *mean = m;
  *rinv = 1.f / sqrtf(block_sum_(q, red) / static_cast<float>(W) + eps);
}

template <int E> __device__ __forceinline__ void ld_row(const float* p, int i, float (&v)[E]) {
  if constexpr (E == 4) {
    const float4 t = reinterpret_cast<const float4*>(p)[i];
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  } else {
    v[0] = p[i];
  }
}

template <typename OT, bool VEC, int NV>
__global__ void __launch_bounds__(1024)
    sandwich_join_kernel(float* __restrict__ x, const int* __restrict__ rows, const float* __restrict__ y, int ld_y, int kind_y,
                         const float* __restrict__ wy, const float* __restrict__ by, int kind_h, const float* __restrict__ wh,
                         const float* __restrict__ bh, float eps, OT* __restrict__ h, int ld_h, int W) {
  constexpr int E = VEC ? 4 : 1;
  __shared__ float red[32];
  const int nv = W / E, nt = blockDim.x;
  pdl_begin();
  const size_t r = blockIdx.x, t = rows != nullptr ? static_cast<size_t>(rows[r]) : r;
  float* xr = x + t * W;
  float v[NV][E];
  float m, ri;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = k * nt + threadIdx.x;
#pragma unroll
    for (int e = 0; e < E; ++e) v[k][e] = 0.f;
    if (i < nv) ld_row<E>(y != nullptr ? y + t * ld_y : xr, i, v[k]);
  }
  if (y != nullptr) {
    float xv[NV][E];
#pragma unroll
    for (int k = 0; k < NV; ++k) {                            // (in flight while the statistics of y are taken)
      const int i = k * nt + threadIdx.x;
      if (i < nv) ld_row<E>(xr, i, xv[k]);
    }
    row_stats<E, NV>(v, nv, W, kind_y, eps, red, &m, &ri);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = k * nt + threadIdx.x;
      if (i >= nv) continue;
      float w[E], b[E];
      ld_row<E>(wy, i, w);
#pragma unroll
      for (int e = 0; e < E; ++e) b[e] = 0.f;
      if (by != nullptr) ld_row<E>(by, i, b);
#pragma unroll
      for (int e = 0; e < E; ++e) v[k][e] = xv[k][e] + ((v[k][e] - m) * ri * w[e] + b[e]);
      if (rows == nullptr) {
        if constexpr (VEC) reinterpret_cast<float4*>(xr)[i] = make_float4(v[k][0], v[k][1], v[k][2], v[k][3]);
        else xr[i] = v[k][0];
      }
    }
  }
  if (h == nullptr) return;
  m = 0.f;
  ri = 1.f;
  if (kind_h != NORM_NONE) row_stats<E, NV>(v, nv, W, kind_h, eps, red, &m, &ri);
  OT* hr = h + r * ld_h;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = k * nt + threadIdx.x;
    if (i >= nv) continue;
    float w[E], b[E];
#pragma unroll
    for (int e = 0; e < E; ++e) {
      w[e] = 1.f;
      b[e] = 0.f;
    }
    if (kind_h != NORM_NONE) {
      ld_row<E>(wh, i, w);
      if (bh != nullptr) ld_row<E>(bh, i, b);
    }
#pragma unroll
    for (int e = 0; e < E; ++e) w[e] = (v[k][e] - m) * ri * w[e] + b[e];
    if constexpr (VEC) st4(hr + 4 * i, make_float4(w[0], w[1], w[2], w[3]));
    else stf(hr, i, w[0]);
  }
}

// ------------------------------------------------------------------------------------------- rotary table
// tab[t, i] = (cos, sin) of positions[t] * (freq[i] + freq_lo[i]), both times amp
__global__ void rot_table_kernel(const int* __restrict__ positions, const float* __restrict__ freq,
                                 const float* __restrict__ freq_lo, int pairs, float amp, float2* __restrict__ tab, int T) {
  pdl_begin();
  const long long e = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (e >= static_cast<long long>(T) * pairs) return;
  const int t = static_cast<int>(e / pairs), i = static_cast<int>(e % pairs);
  float sn, cs;
  turn_(static_cast<float>(positions[t]), freq[i], freq_lo[i], &sn, &cs);
  tab[e] = make_float2(cs * amp, sn * amp);
}

// ------------------------------------------------------------------------------------------- convolution + rotation + cache
// Columns off .. off + C of proj [T, ld] fp32 hold Hq query heads and Gk key heads of D channels and Gv value heads of V
// channels (Gk = Gv = 0: a layer that uses another layer's keys and values).  Every channel passes its own causal convolution
// (w [C, taps], last tap = current token; inputs in front of the span come from tail [slots, taps - 1, C], zeros in front of the
// sequence); channels i and i + half (i < half) of every query and key head turn by the token's table entry i.  Queries are
// multiplied by qscale and go to q_out [T, Hq * D], keys and values to the cache rows of the token's slot.
// A thread owns two channels (a rotary pair, or two adjacent ones) and walks `tpt` tokens with the window in registers.
// DEC: every span is one token; the thread that owns a channel also shifts its tail (spans: conv_commit runs behind).
struct ConvRotArgs {
  const float* proj;
  const float* w;
  float* tail;
  const float2* tab;          // [T, half]
  const int* slots;
  const int* q_start; const int* q_len; const int* kv_len; const int* seq_slot;
  int ld, off, half, Hq, Gk, Gv, D, V, C, taps, tpt;
  float qscale;
};

template <typename QT, typename CT, bool DEC, int MT>
__global__ void __launch_bounds__(128)
    conv_rot_prep_kernel(const ConvRotArgs a, QT* __restrict__ q_out, CT* __restrict__ k_cache, CT* __restrict__ v_cache) {
  pdl_begin();
  const int s = blockIdx.z, n = a.q_len[s];
  const int i0 = blockIdx.y * a.tpt;
  if (i0 >= n) return;
  int u = blockIdx.x * blockDim.x + threadIdx.x;
  const int U = a.half + (a.D - 2 * a.half + 1) / 2, UV = (a.V + 1) / 2, nqk = (a.Hq + a.Gk) * U;
  if (u >= nqk + a.Gv * UV) return;
  int c0, c1, pair = -1, role = 2;                            // role: 0 query, 1 key, 2 value
  bool two = true;
  if (u < nqk) {
    const int sub = u / U, r = u - sub * U;
    role = sub < a.Hq ? 0 : 1;
    if (r < a.half) {
      c0 = sub * a.D + r;
      c1 = c0 + a.half;
      pair = r;
    } else {
      const int d = 2 * a.half + 2 * (r - a.half);
      c0 = sub * a.D + d;
      c1 = c0 + 1;
      two = d + 1 < a.D;
    }
  } else {
    u -= nqk;
    const int hd = u / UV, d = 2 * (u - hd * UV);
    c0 = (a.Hq + a.Gk) * a.D + hd * a.V + d;
    c1 = c0 + 1;
    two = d + 1 < a.V;
  }
  if (!two) c1 = c0;
  const int t0 = a.q_start[s], pos0 = a.kv_len[s] - n, taps = a.taps;
  float* tl = a.tail + static_cast<size_t>(a.seq_slot[s]) * (taps - 1) * a.C;
  const float* x = a.proj + a.off;
  float w0[MT], w1[MT], p0[MT], p1[MT];                       // p[j]: input at distance taps - 1 - j behind the current token
#pragma unroll
  for (int j = 0; j < MT; ++j) {
    w0[j] = w1[j] = p0[j] = p1[j] = 0.f;
    if (j < taps) {
      w0[j] = a.w[static_cast<size_t>(c0) * taps + j];
      w1[j] = a.w[static_cast<size_t>(c1) * taps + j];
    }
    if (j < taps - 1) {
      const int i = i0 - (taps - 1) + j;                      // span index of that input
      if (i >= 0) {
        p0[j] = x[static_cast<size_t>(t0 + i) * a.ld + c0];
        p1[j] = x[static_cast<size_t>(t0 + i) * a.ld + c1];
      } else if (pos0 > 0) {
        p0[j] = tl[static_cast<size_t>(taps - 1 + i) * a.C + c0];
        p1[j] = tl[static_cast<size_t>(taps - 1 + i) * a.C + c1];
      }
    }
  }
  const int i1 = min(n, i0 + a.tpt), nq = a.Hq * a.D;
  for (int i = i0; i < i1; ++i) {
    const size_t t = static_cast<size_t>(t0 + i);
    const float x0 = x[t * a.ld + c0], x1 = x[t * a.ld + c1];
    float y0 = 0.f, y1 = 0.f;
#pragma unroll
    for (int j = 0; j < MT; ++j) {
      if (j < taps - 1) {
        y0 += w0[j] * p0[j];
        y1 += w1[j] * p1[j];
        p0[j] = (j + 1 < MT && j + 1 < taps - 1) ? p0[j + 1 < MT ? j + 1 : j] : x0;
        p1[j] = (j + 1 < MT && j + 1 < taps - 1) ? p1[j + 1 < MT ? j + 1 : j] : x1;
      } else if (j == taps - 1) {
        y0 += w0[j] * x0;
        y1 += w1[j] * x1;
      }
    }
    if (pair >= 0) {
      const float2 cs = a.tab[t * a.half + pair];
      const float r0 = y0 * cs.x - y1 * cs.y;
      y1 = y1 * cs.x + y0 * cs.y;
      y0 = r0;
    }
    if (role == 0) {
      stf(q_out, t * nq + c0, y0 * a.qscale);
      if (two) stf(q_out, t * nq + c1, y1 * a.qscale);
    } else {
      const int slot = a.slots[t];
      if (slot >= 0) {
        CT* dst = role == 1 ? k_cache : v_cache;
        const int nr = role == 1 ? a.Gk * a.D : a.Gv * a.V, cb = role == 1 ? nq : nq + a.Gk * a.D;
        stf(dst, static_cast<size_t>(slot) * nr + (c0 - cb), y0);
        if (two) stf(dst, static_cast<size_t>(slot) * nr + (c1 - cb), y1);
      }
    }
  }
  if (DEC) {                                                  // p now holds the last taps - 1 inputs
#pragma unroll
    for (int j = 0; j < MT; ++j) {
      if (j < taps - 1) {
        tl[static_cast<size_t>(j) * a.C + c0] = p0[j];
        if (two) tl[static_cast<size_t>(j) * a.C + c1] = p1[j];
      }
    }
  }
}

// ------------------------------------------------------------------------------------------- rotated bf16 rows of a recurrence
// columns off .. of proj: H2 heads of D channels (queries, then keys) whose first rdims channels turn in adjacent pairs (2i, 2i + 1) by
// tab [T, rdims] -> qk [T, H2 * D]; columns off_v .. off_v + nv -> v [T, nv].  Four columns per thread (D and nv multiples of 4).
__global__ void __launch_bounds__(256)
    rot_cast_kernel(const float* __restrict__ proj, int ld, int off, int off_v, const float* __restrict__ tab, int rdims,
                    const int* __restrict__ slots, bf16* __restrict__ qk, bf16* __restrict__ v, int H2, int D, int nv) {
  pdl_begin();
  const size_t t = blockIdx.y;
  const int c = (blockIdx.x * 256 + threadIdx.x) * 4, nqk = H2 * D;
  if (c >= nqk + nv || slots[t] < 0) return;
  if (c >= nqk) {
    st4(v + t * nv + (c - nqk), *reinterpret_cast<const float4*>(proj + t * ld + off_v + (c - nqk)));
    return;
  }
  float4 x = *reinterpret_cast<const float4*>(proj + t * ld + off + c);
  const int d = c % D;
  if (d < rdims) {
    const float2 a = *reinterpret_cast<const float2*>(tab + t * rdims + d);
    float2 b = make_float2(1.f, 0.f);
    if (d + 2 < rdims) b = *reinterpret_cast<const float2*>(tab + t * rdims + d + 2);
    x = make_float4(x.x * a.x - x.y * a.y, x.y * a.x + x.x * a.y, x.z * b.x - x.w * b.y, x.w * b.x + x.z * b.y);
  }
  st4(qk + t * nqk + c, x);
}

// ------------------------------------------------------------------------------------------- differential attention: the two maps
// in [T, 2 H V] fp32: map outputs in the order (key/value head, map, head of its group); out[t, h, :] = d / rms(d) * gain with
// d = a_1 - lambda a_2.  One warp per (token, head).
template <typename OT>
__global__ void __launch_bounds__(128)
    diff_combine_kernel(const float* __restrict__ in, int ld_in, float lambda, float gain, OT* __restrict__ out, int ld_out, int T,
                        int H, int G, int V, float eps) {
  pdl_begin();
  const long long wid = static_cast<long long>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (wid >= static_cast<long long>(T) * H) return;
  const size_t t = static_cast<size_t>(wid / H);
  const int hd = static_cast<int>(wid % H), r = H / G, g = hd / r, i = hd - g * r;
  const float* a = in + t * ld_in + static_cast<size_t>(2 * g * r + i) * V;
  const float* b = a + static_cast<size_t>(r) * V;
  float ss = 0.f;
  for (int d = lane; d < V; d += 32) {
    const float v = a[d] - lambda * b[d];
    ss += v * v;
  }
  const float k = gain / sqrtf(warp_sum_(ss) / static_cast<float>(V) + eps);
  for (int d = lane; d < V; d += 32) stf(out, t * ld_out + static_cast<size_t>(hd) * V + d, (a[d] - lambda * b[d]) * k);
}

// ------------------------------------------------------------------------------------------- state-space output
// out[t, c] = v / rms(part of c) * w[c] with v = (o[t, c] + skip[c / V] x[t, c]) * silu(z[t, c]), c < n = heads * V, the root mean
// square taken over `parts` equal consecutive parts.  One block per (token, part); the part is kept in shared memory.
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename OT, typename XT, bool VEC>
__global__ void __launch_bounds__(256)
    ssd_post_kernel(const float* __restrict__ o, int ld_o, const XT* __restrict__ x, int ld_x, const float* __restrict__ z, int ld_z,
                    const float* __restrict__ skip, const float* __restrict__ w, OT* __restrict__ out, int ld_out, int n, int V,
                    int parts, float eps) {
  pdl_begin();
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  const size_t t = blockIdx.x;
  const int np = n / parts, c0 = blockIdx.y * np;
  const float* orow = o + t * ld_o + c0;
  const XT* xrow = x + t * ld_x + c0;
  const float* zrow = z + t * ld_z + c0;
  float ss = 0.f;
  if constexpr (VEC) {
    for (int c = 4 * threadIdx.x; c < np; c += 4 * blockDim.x) {
      const float4 ov = *reinterpret_cast<const float4*>(orow + c), xv = ld4(xrow + c),
                   zv = *reinterpret_cast<const float4*>(zrow + c);
      const float D = skip[(c0 + c) / V];
      const float4 v = make_float4((ov.x + D * xv.x) * silu_(zv.x), (ov.y + D * xv.y) * silu_(zv.y), (ov.z + D * xv.z) * silu_(zv.z),
                                   (ov.w + D * xv.w) * silu_(zv.w));
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      *reinterpret_cast<float4*>(row + c) = v;
    }
  } else {
    for (int c = threadIdx.x; c < np; c += blockDim.x) {
      const float v = (orow[c] + skip[(c0 + c) / V] * ldf(xrow, c)) * silu_(zrow[c]);
      ss += v * v;
      row[c] = v;
    }
  }
  const float r = 1.f / sqrtf(block_sum_(ss, red) / static_cast<float>(np) + eps);
  OT* dst = out + t * ld_out + c0;
  if constexpr (VEC) {
    for (int c = 4 * threadIdx.x; c < np; c += 4 * blockDim.x) {
      const float4 v = *reinterpret_cast<const float4*>(row + c), g = *reinterpret_cast<const float4*>(w + c0 + c);
      st4(dst + c, make_float4(v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w));
    }
  } else {
    for (int c = threadIdx.x; c < np; c += blockDim.x) stf(dst, c, row[c] * r * w[c0 + c]);
  }
}

// ------------------------------------------------------------------------------------------- per-token channels
// out[t, c] = gelu_tanh(z[t, c]) * table[ids[t], off + c], c < n
template <typename OT>
__global__ void side_gate_kernel(const float* __restrict__ z, int ld_z, const int* __restrict__ ids, const OT* __restrict__ table,
                                 int ld_t, int off, int vocab, OT* __restrict__ out, int ld_out, int n, int T) {
  pdl_begin();
  const long long e = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (e >= static_cast<long long>(T) * n) return;
  const int c = static_cast<int>(e % n);
  const size_t t = static_cast<size_t>(e / n);
  const int id = min(max(ids[t], 0), vocab - 1);
  stf(out, t * ld_out + c, gelu_tanh_(z[t * ld_z + c]) * ldf(table, static_cast<size_t>(id) * ld_t + off + c));
}

inline int last_error() { return static_cast<int>(cudaGetLastError()); }
inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

int launch_sandwich_join(float* x, const int* rows, int n_rows, const float* y, int ld_y, int kind_y, const float* wy,
                         const float* by, int kind_h, const float* wh, const float* bh, float eps, void* h, int ld_h, int W, int f32,
                         cudaStream_t s) {
  if (n_rows <= 0) return 0;
  if (y != nullptr && (wy == nullptr || kind_y > NORM_LAYER)) return -2;
  if (h != nullptr && kind_h != NORM_NONE && wh == nullptr) return -2;
  const bool vec = W % 4 == 0 && al16(x) && al16(y) && al16(wy) && al16(by) && al16(wh) && al16(bh) && al16(h) && ld_y % 4 == 0 &&
                   ld_h % 4 == 0;
  const int nv = vec ? W / 4 : W;
  int threads = (nv + 31) / 32 * 32;
  const int cap = n_rows <= 296 ? 512 : 256;                 // few rows (decode steps): more threads per row
  if (threads > cap) threads = cap;
  while (threads < 1024 && (nv + threads - 1) / threads > 16) threads = threads * 2 < 1024 ? threads * 2 : 1024;
  const int per = (nv + threads - 1) / threads;
  if (per > 16) return -2;
#define B2B_SJ(OT, VEC, NV)                                                                                              \
  launch_kernel(sandwich_join_kernel<OT, VEC, NV>, dim3(n_rows), dim3(threads), 0, s, 1u, x, rows, y, ld_y, kind_y, wy, by, \
                kind_h, wh, bh, eps, static_cast<OT*>(h), ld_h, W)
#define B2B_SJ_T(OT, VEC)                                                                                                \
  do {                                                                                                                   \
    if (per <= 1) B2B_SJ(OT, VEC, 1);                                                                                    \
    else if (per <= 2) B2B_SJ(OT, VEC, 2);                                                                               \
    else if (per <= 4) B2B_SJ(OT, VEC, 4);                                                                               \
    else if (per <= 8) B2B_SJ(OT, VEC, 8);                                                                               \
    else B2B_SJ(OT, VEC, 16);                                                                                            \
  } while (0)
  if (f32) {
    if (vec) B2B_SJ_T(float, true);
    else B2B_SJ_T(float, false);
  } else {
    if (vec) B2B_SJ_T(bf16, true);
    else B2B_SJ_T(bf16, false);
  }
#undef B2B_SJ_T
#undef B2B_SJ
  return last_error();
}

int launch_rot_table(const int* positions, const float* freq, const float* freq_lo, int pairs, float amp, float* tab, int T,
                     cudaStream_t s) {
  const long long n = static_cast<long long>(T) * pairs;
  if (n <= 0) return 0;
  launch_kernel(rot_table_kernel, dim3(static_cast<unsigned>((n + 127) / 128)), dim3(128), 0, s, 1u, positions, freq, freq_lo, pairs,
                amp, reinterpret_cast<float2*>(tab), T);
  return last_error();
}

int launch_conv_rot_prep(const float* proj, int ld, int off, const float* w, float* tail, const float* tab, int half, float qscale,
                         const int* slots, void* q_out, int q_f32, void* k_cache, void* v_cache, int c_f32, const int* q_start,
                         const int* q_len, const int* kv_len, const int* seq_slot, int n_seqs, int max_q, int Hq, int Gk, int Gv,
                         int D, int V, int taps, cudaStream_t s) {
  if (n_seqs <= 0 || max_q <= 0) return 0;
  if (taps < 1 || taps > 32 || 2 * half > D || (c_f32 && !q_f32)) return -2;
  ConvRotArgs a{proj, w, tail, reinterpret_cast<const float2*>(tab), slots, q_start, q_len, kv_len, seq_slot,
                ld, off, half, Hq, Gk, Gv, D, V, (Hq + Gk) * D + Gv * V, taps, 16, qscale};
  const int U = half + (D - 2 * half + 1) / 2, units = (Hq + Gk) * U + Gv * ((V + 1) / 2);
  const bool dec = max_q == 1;
  const dim3 grid((units + 127) / 128, (max_q + a.tpt - 1) / a.tpt, n_seqs);
#define B2B_CR(QT, CT, DEC, MT)                                                                                          \
  launch_kernel(conv_rot_prep_kernel<QT, CT, DEC, MT>, grid, dim3(128), 0, s, 1u, a, static_cast<QT*>(q_out),            \
                static_cast<CT*>(k_cache), static_cast<CT*>(v_cache))
#define B2B_CR_D(QT, CT)                                                                                                 \
  do {                                                                                                                   \
    if (taps <= 4) {                                                                                                     \
      if (dec) B2B_CR(QT, CT, true, 4);                                                                                  \
      else B2B_CR(QT, CT, false, 4);                                                                                     \
    } else {                                                                                                             \
      if (dec) B2B_CR(QT, CT, true, 32);                                                                                 \
      else B2B_CR(QT, CT, false, 32);                                                                                    \
    }                                                                                                                    \
  } while (0)
  if (c_f32) B2B_CR_D(float, float);
  else if (q_f32) B2B_CR_D(float, bf16);
  else B2B_CR_D(bf16, bf16);
#undef B2B_CR_D
#undef B2B_CR
  if (!dec && taps > 1) {
    const int e = last_error();
    if (e) return e;
    return launch_short_conv_commit(proj, ld, off, tail, q_start, q_len, kv_len, seq_slot, n_seqs, a.C, taps, s);
  }
  return last_error();
}

int launch_rot_cast(const float* proj, int ld, int off, int off_v, const float* tab, int rdims, const int* slots, void* qk, void* v, int T,
                    int H2, int D, int nv, cudaStream_t s) {
  if (T <= 0) return 0;
  if (D % 4 != 0 || nv % 4 != 0 || ld % 4 != 0 || off % 4 != 0 || off_v % 4 != 0 || !al16(proj) || rdims % 2 != 0 || rdims > D || T > 65535) return -2;
  const int cols = H2 * D + nv;
  launch_kernel(rot_cast_kernel, dim3((cols / 4 + 255) / 256, T), dim3(256), 0, s, 1u, proj, ld, off, off_v, tab, rdims, slots,
                static_cast<bf16*>(qk), static_cast<bf16*>(v), H2, D, nv);
  return last_error();
}

int launch_diff_combine(const float* in, int ld_in, float lambda, float gain, void* out, int ld_out, int T, int H, int G, int V,
                        float eps, int f32, cudaStream_t s) {
  const long long warps = static_cast<long long>(T) * H;
  if (warps <= 0) return 0;
  if (G <= 0 || H % G != 0) return -2;
  const dim3 grid(static_cast<unsigned>((warps + 3) / 4));
  if (f32)
    launch_kernel(diff_combine_kernel<float>, grid, dim3(128), 0, s, 1u, in, ld_in, lambda, gain, static_cast<float*>(out), ld_out, T, H,
                  G, V, eps);
  else
    launch_kernel(diff_combine_kernel<bf16>, grid, dim3(128), 0, s, 1u, in, ld_in, lambda, gain, static_cast<bf16*>(out), ld_out, T, H,
                  G, V, eps);
  return last_error();
}

int launch_ssd_post(const float* o, int ld_o, const void* x, int x_f32, int ld_x, const float* z, int ld_z, const float* skip, const float* w,
                    void* out, int ld_out, int T, int H, int V, int parts, float eps, int f32, cudaStream_t s) {
  const int n = H * V;
  if (T <= 0 || n <= 0) return 0;
  if (parts <= 0 || n % parts != 0 || parts > 65535) return -2;
  const int np = n / parts;
  const size_t smem = static_cast<size_t>(np) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  const bool vec = V % 4 == 0 && np % 4 == 0 && ld_o % 4 == 0 && ld_x % 4 == 0 && ld_z % 4 == 0 && ld_out % 4 == 0 && al16(o) && al16(x) &&
                   al16(z) && al16(w) && al16(out);
  int threads = ((vec ? np / 4 : np) + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  if (f32 && !x_f32) return -2;
#define B2B_SP(OT, XT, VEC)                                                                                              \
  do {                                                                                                                   \
    if (smem > 48 * 1024)                                                                                                \
      cudaFuncSetAttribute(ssd_post_kernel<OT, XT, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)); \
    launch_kernel(ssd_post_kernel<OT, XT, VEC>, dim3(T, parts), dim3(threads), smem, s, 1u, o, ld_o, static_cast<const XT*>(x), ld_x, z, \
                  ld_z, skip, w, static_cast<OT*>(out), ld_out, n, V, parts, eps);                                       \
  } while (0)
  if (f32) {
    if (vec) B2B_SP(float, float, true);
    else B2B_SP(float, float, false);
  } else if (x_f32) {
    if (vec) B2B_SP(bf16, float, true);
    else B2B_SP(bf16, float, false);
  } else {
    if (vec) B2B_SP(bf16, bf16, true);
    else B2B_SP(bf16, bf16, false);
  }
#undef B2B_SP
  return last_error();
}

int launch_side_gate(const float* z, int ld_z, const int* ids, const void* table, int ld_t, int off, int vocab, void* out, int ld_out,
                     int n, int T, int f32, cudaStream_t s) {
  const long long tot = static_cast<long long>(T) * n;
  if (tot <= 0) return 0;
  const dim3 grid(static_cast<unsigned>((tot + 127) / 128));
  if (f32)
    launch_kernel(side_gate_kernel<float>, grid, dim3(128), 0, s, 1u, z, ld_z, ids, static_cast<const float*>(table), ld_t, off, vocab,
                  static_cast<float*>(out), ld_out, n, T);
  else
    launch_kernel(side_gate_kernel<bf16>, grid, dim3(128), 0, s, 1u, z, ld_z, ids, static_cast<const bf16*>(table), ld_t, off, vocab,
                  static_cast<bf16*>(out), ld_out, n, T);
  return last_error();
}

}  // namespace b2b
