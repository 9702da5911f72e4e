// Linear recurrences with ONE decay per head and token: lin_chunk runs whole chunks of a span on tensor cores (bf16 serving mode),
// lin_step single tokens of many sequences as a stream over their states (below); short spans and long spans of the float32 mode walk
// token by token in lin_scan, seqmix.cu.  All of them work on the same fp32 states:
//     S_t = d_t S_(t-1) + b_t k_t v_t^T,   o_t = qscale S_t^T q_t          (S [dk, dv] per head and sequence slot)
//   state-space   d_t = exp(-exp(A_h) b_t), b_t = softplus(x_t + bias_h)    (q / k of a group of heads)
//   retention     d_t = decay_h, b_t = 1
// With c_t = log d_1 + ... + log d_t inside a chunk of 64 tokens that starts from S_0:
//     o_t = qscale (exp(c_t) S_0^T q_t + sum_(s <= t) exp(c_t - c_s) b_s (q_t . k_s) v_s)
//     S_L = exp(c_L) S_0 + sum_s exp(c_L - c_s) b_s k_s v_s^T
// so a chunk is four matrix products instead of 64 dependent steps.  q, k and v are bf16 (projections and convolved activations);
// everything that enters the recurrence besides them keeps fp32 precision: decays, their logarithms and sums, step sizes, the
// state (fp32 accumulators that stay in registers from chunk to chunk), and where a product of such numbers is an operand (weighted
// scores, weighted values, the state in front of q) it is split into a high and a low bf16 part, 16 bits of mantissa together.
// A block = 32 state columns of one (sequence, head), sixteen warps.  Tokens of the chunk are the M dimension of the output products
// (four tiles of 16, four warps each that split the keys and the state rows); state rows are the M dimension of the update.
// The next chunk's rows come in by cp.async meanwhile, and one warp prepares its decays and step sizes.
// This translation unit is compiled WITHOUT --use_fast_math (exact expf / logf / softplus); the weights inside a chunk are the
// hardware exp2 (2^-22 relative).
#include "kernels.h"

#include <cuda_bf16.h>

#include <cstdint>

#include "common.cuh"
#include "launch.cuh"
#include "tmem.cuh"

namespace b2b {
namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ void pdl_begin() {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
}
__device__ __forceinline__ float softplus_(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ uint32_t sptr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool take) {      // !take: zeros
  const int n = take ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
// two numbers as packed bf16 pairs: high parts, and what the high parts leave over
__device__ __forceinline__ void split2(float x, float y, uint32_t* hi, uint32_t* lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  *hi = *reinterpret_cast<const uint32_t*>(&h);
  *lo = *reinterpret_cast<const uint32_t*>(&l);
}

constexpr int LC_L = 64, LC_VB = 32, LC_WARPS = 16, LC_THREADS = 32 * LC_WARPS;
constexpr int LC_VS = LC_VB + 8;                       // row stride of value and state tiles (elements)
constexpr int LC_OS = LC_VB + 8;                       // row stride of partial outputs (floats)

// partial outputs that go through shared memory: all four of a token tile, or (widest states: no room) three beside one in registers
__host__ __device__ constexpr int lc_parts(int KT) { return KT > 8 ? 3 : 4; }

struct ChunkArgs {
  const bf16* q; const bf16* k; const bf16* v;         // [T, ld] rows, already at their first column
  int ld_q, ld_k, ld_v;
  const float* step; int ld_step;                      // state-space: step size before bias and softplus, column of head 0
  const float* bias;                                   // [H]
  const float* hparam;                                 // state-space: A_log [H]; retention: decay [H]
  float qscale;
  float* state; float* out; int ld_out;
  const int* q_start; const int* q_len; const int* kv_len; const int* seq_slot;
  int H, G, dk, dv;
};

// KT: dk in units of 16, rounded up to an instance (dk <= 16 KT, zero padded).  SSD: state-space, otherwise retention.
template <int KT, bool SSD>
__global__ void __launch_bounds__(LC_THREADS, 1)
    lin_chunk_kernel(const ChunkArgs a) {
  pdl_begin();
  constexpr int NP = 16 * KT, RS = NP + 8;             // row stride of q / k tiles
  constexpr int UN = KT > 8 ? KT / 8 : 1;              // state units (16 rows x 16 columns) per warp
  constexpr int TILE = LC_L * RS, VT = LC_L * LC_VS, OB = lc_parts(KT);
  constexpr float LOG2E = 1.4426950408889634f;
  extern __shared__ __align__(16) uint8_t smem_[];
  bf16* qs = reinterpret_cast<bf16*>(smem_);           // [2][64][RS]
  bf16* ks = qs + 2 * TILE;
  bf16* vs = ks + 2 * TILE;                            // [2][64][VS]
  bf16* sh = vs + 2 * VT;                              // [NP][VS] state, high parts
  bf16* sl = sh + NP * LC_VS;
  bf16* vh = sl + NP * LC_VS;                          // [64][VS] values times their weight in the update, high and low parts
  bf16* vl = vh + VT;
  float* ox = reinterpret_cast<float*>(vl + VT);       // [4][64][OS] partial outputs of the four warps of a token tile
  float* scal = ox + OB * LC_L * LC_OS;                 // [2][3][64]: c_t (in powers of two), b_s, exp(c_L - c_s) b_s
  const int s = blockIdx.z, hd = blockIdx.y, v0 = blockIdx.x * LC_VB;
  const int n = a.q_len[s];
  if (n <= 0) return;                                  // (block-uniform)
  const int t0 = a.q_start[s], pos0 = a.kv_len[s] - n;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;
  const int hq = SSD ? hd / (a.H / a.G) : hd;
  const bf16* qg = a.q + static_cast<size_t>(hq) * a.dk;
  const bf16* kg = a.k + static_cast<size_t>(hq) * a.dk;
  const bf16* vg = a.v + static_cast<size_t>(hd) * a.dv + v0;
  float* Sg = a.state + (static_cast<size_t>(a.seq_slot[s]) * a.H + hd) * static_cast<size_t>(a.dk) * a.dv + v0;

  // state units of this warp: unit = warp + 16 u -> rows (unit % KT) * 16 .., columns (unit / KT) * 16 ..
  const bool owner = warp < 2 * KT;
  float S[UN][2][4];
  auto s_row = [&](int u, int e) { return (warp + LC_WARPS * u) % KT * 16 + gid + (e >> 1) * 8; };
  auto s_col = [&](int u, int nt) { return (warp + LC_WARPS * u) / KT * 16 + nt * 8 + 2 * tig; };
#pragma unroll
  for (int u = 0; u < UN; ++u)
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = s_row(u, e), c = s_col(u, nt) + (e & 1);
        S[u][nt][e] = (owner && pos0 > 0 && r < a.dk && v0 + c < a.dv) ? Sg[static_cast<size_t>(r) * a.dv + c] : 0.f;
      }

  // this thread's pieces of a chunk: q and k rows sr[] (16 bytes at column sc), and (first 256 threads) 8 channels of value row tid / 4
  constexpr int PC = (LC_L * (NP / 8) + LC_THREADS - 1) / LC_THREADS;
  const int sr = tid / (NP / 8), scol = tid % (NP / 8) * 8, vr = tid >> 2, vc = (tid & 3) * 8;
  constexpr int STEP = LC_THREADS / (NP / 8);          // rows between two pieces of a thread
  const bool s_ok = scol < a.dk, v_ok = tid < 4 * LC_L && v0 + vc < a.dv;
  const bf16* qp = qg + static_cast<size_t>(t0 + sr) * a.ld_q + scol;
  const bf16* kp = kg + static_cast<size_t>(t0 + sr) * a.ld_k + scol;
  const bf16* vp = vg + static_cast<size_t>(t0 + vr) * a.ld_v + vc;
  const uint32_t qd = sptr(qs + sr * RS + scol), kd = sptr(ks + sr * RS + scol), vd = sptr(vs + vr * LC_VS + vc);
  auto stage = [&](int ch) {                           // (called once per chunk, in order)
    const int left = n - ch * LC_L;
    const uint32_t bq = (ch & 1) * TILE * 2;
#pragma unroll
    for (int i = 0; i < PC; ++i) {
      const bool ok = s_ok && sr + i * STEP < left;
      cp16(qd + bq + i * STEP * RS * 2, ok ? qp + i * STEP * a.ld_q : a.q, ok);
      cp16(kd + bq + i * STEP * RS * 2, ok ? kp + i * STEP * a.ld_k : a.k, ok);
    }
    if (tid < 4 * LC_L) {
      const bool ok = v_ok && vr < left;
      cp16(vd + (ch & 1) * VT * 2, ok ? vp : a.v, ok);
    }
    qp += static_cast<size_t>(LC_L) * a.ld_q;
    kp += static_cast<size_t>(LC_L) * a.ld_k;
    vp += static_cast<size_t>(LC_L) * a.ld_v;
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  // the scalar part of a chunk, by one warp that has no keys in front of its tokens (two tokens per lane): step sizes, decays, sums
  constexpr int SW = 12;
  const float rate = SSD ? expf(a.hparam[hd]) : 0.f, bias = SSD ? a.bias[hd] : 0.f;
  const float logd = SSD ? 0.f : fmaxf(logf(a.hparam[hd]), -80.f);      // (a decay of zero: exp(-80) is zero beside any other term)
  auto load_step = [&](int ch, float* x) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = ch * LC_L + 2 * lane + e;
      x[e] = (SSD && i < n) ? a.step[static_cast<size_t>(t0 + i) * a.ld_step + hd] : 0.f;
    }
  };
  auto scalars = [&](int ch, const float* x) {
    float* sc = scal + (ch & 1) * 3 * LC_L;
    float b[2], lg[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool in = ch * LC_L + 2 * lane + e < n;
      b[e] = in ? (SSD ? softplus_(x[e] + bias) : 1.f) : 0.f;
      lg[e] = SSD ? -rate * b[e] : (in ? logd : 0.f);
    }
    float run = lg[0] + lg[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float u = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += u;
    }
    const float before = run - lg[1], last = __shfl_sync(0xffffffffu, run, 31);
    *reinterpret_cast<float2*>(sc + 2 * lane) = make_float2(before * LOG2E, run * LOG2E);
    *reinterpret_cast<float2*>(sc + LC_L + 2 * lane) = make_float2(b[0], b[1]);
    *reinterpret_cast<float2*>(sc + 2 * LC_L + 2 * lane) = make_float2(expf(last - before) * b[0], expf(last - run) * b[1]);
  };

  const int nch = (n + LC_L - 1) / LC_L;
  stage(0);
  float xs[2] = {0.f, 0.f};
  if (warp == SW) {
    load_step(0, xs);
    scalars(0, xs);
    if (nch > 1) load_step(1, xs);
  }
  __syncthreads();
  const int mt = warp & 3, kh = warp >> 2;             // token tile; which quarter of the keys and of the state rows
  const uint32_t vt_off = (((lane & 7) + ((lane >> 3) & 1) * 8) * LC_VS + (lane >> 4) * 8) * 2;
  for (int ch = 0; ch < nch; ++ch) {
    const int buf = ch & 1, tb = ch * LC_L;
    if (ch + 1 < nch) stage(ch + 1);
    else asm volatile("cp.async.commit_group;\n" ::: "memory");
    if (owner) {                                       // the state in front of this chunk as an operand
#pragma unroll
      for (int u = 0; u < UN; ++u)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            uint32_t hi, lo;
            split2(S[u][nt][2 * e], S[u][nt][2 * e + 1], &hi, &lo);
            *reinterpret_cast<uint32_t*>(sh + s_row(u, 2 * e) * LC_VS + s_col(u, nt)) = hi;
            *reinterpret_cast<uint32_t*>(sl + s_row(u, 2 * e) * LC_VS + s_col(u, nt)) = lo;
          }
    }
    asm volatile("cp.async.wait_group 1;\n" ::: "memory");
    const float* cum = scal + buf * 3 * LC_L;
    const float* wst = cum + LC_L;
    if (tid < 4 * LC_L) {                              // the values this thread has copied, weighted for the update
      const float w = wst[LC_L + vr];
      const uint4 x = *reinterpret_cast<const uint4*>(vs + buf * VT + vr * LC_VS + vc);
      const uint32_t xw[4] = {x.x, x.y, x.z, x.w};
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&xw[e]));
        split2(f.x * w, f.y * w, &hi[e], &lo[e]);
      }
      *reinterpret_cast<uint4*>(vh + vr * LC_VS + vc) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(vl + vr * LC_VS + vc) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    __syncthreads();

    // ---- outputs of 16 tokens against a quarter of the keys and of the state rows
    float op[4][4], os[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) op[i][e] = os[i][e] = 0.f;
    const int r0 = mt * 16 + gid, r1 = r0 + 8;
    const float cr0 = cum[r0], cr1 = cum[r1];
    const uint32_t qa = sptr(qs + buf * TILE + (mt * 16 + (lane & 15)) * RS + (lane >> 4) * 8);
    const bool seen = kh <= mt;                        // (keys behind every token of the tile: nothing)
    float g[4][4];                                     // two key tiles, even and odd steps apart (shorter chains)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) g[i][e] = 0.f;
    {
      const uint32_t ha = sptr(sh) + vt_off, la = sptr(sl) + vt_off;
      const uint32_t kb = sptr(ks + buf * TILE + (kh * 16 + (lane & 7) + (lane >> 4) * 8) * RS + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int kk = 0; kk < KT; ++kk) {
        const bool mine = kk / (KT / 4) == kh;         // this warp's quarter of the state rows
        if (!seen && !mine) continue;
        uint32_t af[4];
        ldsm(af, qa + kk * 32);
        if (seen) {
          uint32_t b[4];
          ldsm(b, kb + kk * 32);
          mma(g[2 * (kk & 1)], af, b[0], b[1]);
          mma(g[2 * (kk & 1) + 1], af, b[2], b[3]);
        }
        if (mine) {
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            uint32_t b[4], d[4];
            ldsm_t(b, ha + kk * 16 * LC_VS * 2 + j * 32);
            ldsm_t(d, la + kk * 16 * LC_VS * 2 + j * 32);
            mma(os[2 * j], af, b[0], b[1]);
            mma(os[2 * j + 1], af, b[2], b[3]);
            mma(os[2 * j], af, d[0], d[1]);
            mma(os[2 * j + 1], af, d[2], d[3]);
          }
        }
      }
    }
    if (seen) {
      // weighted scores -> A operand (high, low), times the values
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int c = kh * 16 + h * 8 + 2 * tig;
        const float2 cc = *reinterpret_cast<const float2*>(cum + c), ww = *reinterpret_cast<const float2*>(wst + c);
        const float p00 = c <= r0 ? (g[h][0] + g[h + 2][0]) * ex2(cr0 - cc.x) * ww.x : 0.f;
        const float p01 = c + 1 <= r0 ? (g[h][1] + g[h + 2][1]) * ex2(cr0 - cc.y) * ww.y : 0.f;
        const float p10 = c <= r1 ? (g[h][2] + g[h + 2][2]) * ex2(cr1 - cc.x) * ww.x : 0.f;
        const float p11 = c + 1 <= r1 ? (g[h][3] + g[h + 2][3]) * ex2(cr1 - cc.y) * ww.y : 0.f;
        split2(p00, p01, &ph[2 * h], &pl[2 * h]);
        split2(p10, p11, &ph[2 * h + 1], &pl[2 * h + 1]);
      }
      const uint32_t va = sptr(vs + buf * VT + kh * 16 * LC_VS) + vt_off;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        uint32_t b[4];
        ldsm_t(b, va + j * 32);
        mma(op[2 * j], ph, b[0], b[1]);
        mma(op[2 * j + 1], ph, b[2], b[3]);
        mma(op[2 * j], pl, b[0], b[1]);
        mma(op[2 * j + 1], pl, b[2], b[3]);
      }
    }
    if (warp == SW && ch + 1 < nch) {
      scalars(ch + 1, xs);
      if (ch + 2 < nch) load_step(ch + 2, xs);
    }
    {
      const float e0 = ex2(cr0), e1 = ex2(cr1);
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) op[nt][e] += (e < 2 ? e0 : e1) * os[nt][e];
      if (OB == 4 || kh > 0) {
        float* dst = ox + ((kh - (4 - OB)) * LC_L + r0) * LC_OS + 2 * tig;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          *reinterpret_cast<float2*>(dst + nt * 8) = make_float2(op[nt][0], op[nt][1]);
          *reinterpret_cast<float2*>(dst + 8 * LC_OS + nt * 8) = make_float2(op[nt][2], op[nt][3]);
        }
      }
    }
    // ---- state behind this chunk: 16 rows x 16 columns per unit, over all tokens
    if (owner) {
      const float dec = ex2(cum[LC_L - 1]);
#pragma unroll
      for (int u = 0; u < UN; ++u)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[u][nt][e] *= dec;
#pragma unroll
      for (int k2 = 0; k2 < LC_L / 16; ++k2) {
#pragma unroll
        for (int u = 0; u < UN; ++u) {
          const int unit = warp + LC_WARPS * u;
          uint32_t kf[4], b[4], d[4];
          ldsm_t(kf, sptr(ks + buf * TILE + (k2 * 16 + (lane & 7) + (lane >> 4) * 8) * RS + unit % KT * 16 + ((lane >> 3) & 1) * 8));
          ldsm_t(b, sptr(vh + k2 * 16 * LC_VS) + vt_off + unit / KT * 32);
          ldsm_t(d, sptr(vl + k2 * 16 * LC_VS) + vt_off + unit / KT * 32);
          mma(S[u][0], kf, b[0], b[1]);
          mma(S[u][1], kf, b[2], b[3]);
          mma(S[u][0], kf, d[0], d[1]);
          mma(S[u][1], kf, d[2], d[3]);
        }
      }
    }
    __syncthreads();                                   // partial outputs are there; tiles and the state operand may be written again
    if constexpr (OB == 3) {
      if (kh == 0) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = r0 + e * 8;
          if (tb + r >= n) continue;
          float* dst = a.out + static_cast<size_t>(t0 + tb + r) * a.ld_out + static_cast<size_t>(hd) * a.dv + v0;
#pragma unroll
          for (int nt = 0; nt < 4; ++nt) {
            const int c = nt * 8 + 2 * tig;
            float2 v = make_float2(op[nt][2 * e], op[nt][2 * e + 1]);
#pragma unroll
            for (int k = 0; k < OB; ++k) {
              const float2 o = *reinterpret_cast<const float2*>(ox + (k * LC_L + r) * LC_OS + c);
              v = make_float2(v.x + o.x, v.y + o.y);
            }
            if (v0 + c < a.dv) *reinterpret_cast<float2*>(dst + c) = make_float2(v.x * a.qscale, v.y * a.qscale);
          }
        }
      }
    } else {
      const int r = tid >> 3, c = (tid & 7) * 4;       // 64 rows x 8 pieces of 4 columns
      if (tb + r < n && v0 + c < a.dv) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float4 o = *reinterpret_cast<const float4*>(ox + (k * LC_L + r) * LC_OS + c);
          v = make_float4(v.x + o.x, v.y + o.y, v.z + o.z, v.w + o.w);
        }
        *reinterpret_cast<float4*>(a.out + static_cast<size_t>(t0 + tb + r) * a.ld_out + static_cast<size_t>(hd) * a.dv + v0 + c) =
            make_float4(v.x * a.qscale, v.y * a.qscale, v.z * a.qscale, v.w * a.qscale);
      }
    }
  }
#pragma unroll
  for (int u = 0; u < UN; ++u)
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = s_row(u, e), c = s_col(u, nt) + (e & 1);
        if (owner && r < a.dk && v0 + c < a.dv) Sg[static_cast<size_t>(r) * a.dv + c] = S[u][nt][e];
      }
}

template <int KT, bool SSD>
int launch_kt(const ChunkArgs& a, int n_seqs, cudaStream_t s) {
  constexpr int NP = 16 * KT, RS = NP + 8;
  constexpr size_t bytes = static_cast<size_t>(4 * LC_L * RS + 4 * LC_L * LC_VS + 2 * NP * LC_VS) * 2 +
                           static_cast<size_t>(lc_parts(KT) * LC_L * LC_OS + 6 * LC_L) * 4;
  static_assert(bytes <= 227 * 1024, "shared memory of a block");
  static bool set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 64 || !set[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(lin_chunk_kernel<KT, SSD>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes));
    if (e != cudaSuccess) return static_cast<int>(e);
    if (dev < 64) set[dev] = true;
  }
  return static_cast<int>(launch_kernel(lin_chunk_kernel<KT, SSD>, dim3((a.dv + LC_VB - 1) / LC_VB, a.H, n_seqs), dim3(LC_THREADS), bytes, s,
                                        1u, a));
}

// ------------------------------------------------------------------------------------------- decode steps: a stream over the states
// Every span is one token.  The [dk, dv] states are contiguous, so a CTA streams them through shared memory with bulk copies: two CTAs
// per SM, each with a ring of row blocks of at most 32 KB; a loader warp fills stages ahead, eight warps update a block in place
// and read it with q, a storer warp sends it back and releases the stage.  The small inputs of the next (sequence, head) are
// fetched while this one is worked on.  Everything is fp32.  Waits are bounded (see tmem.cuh); a CTA whose wait runs out raises
// the engine's abort word, lets its copies land and leaves.
constexpr int LP_STAGES = 3, LP_BYTES = 32 * 1024, LP_WORK = 256, LP_THREADS = LP_WORK + 64;
struct StepArgs {
  const float* q; const float* k; const float* v;      // rows, already at their first column
  int ld_q, ld_k, ld_v;
  const float* step; int ld_step;
  const float* bias;
  const float* hparam;
  const float* tab;                                    // retention: rotary table [T, rdims] of (cos, sin)
  int rdims;
  float qscale;
  float* state; float* out; int ld_out;
  const int* q_start; const int* q_len; const int* kv_len; const int* seq_slot;
  int n_seqs, H, G, dk, dv, rows;                      // rows of a block of the ring
};

__device__ unsigned int g_step_gave_up = 0;            // CTAs whose waits ran out since the module was loaded

template <bool SSD>
__global__ void __launch_bounds__(LP_THREADS)
    lin_step_kernel(const StepArgs a) {
  extern __shared__ __align__(128) uint8_t smem_[];
  float* ring = reinterpret_cast<float*>(smem_);                       // [LP_STAGES][LP_BYTES]
  float* par = ring + LP_STAGES * LP_BYTES / 4;                        // [2][3][256]: weighted k, q, v
  float* sc = par + 2 * 3 * 256;                                       // [2] decay
  float* red = sc + 4;                                                 // [2][LP_WORK * 4] partial outputs
  uint64_t* full = reinterpret_cast<uint64_t*>(red + 2 * LP_WORK * 4);
  uint64_t* done = full + LP_STAGES;
  uint64_t* empty = done + LP_STAGES;
  uint32_t* flags = reinterpret_cast<uint32_t*>(empty + LP_STAGES);
  volatile uint32_t* abort = flags;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int i = 0; i < LP_STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&done[i], LP_WORK / 32);
      mbar_init(&empty[i], 1);
    }
    *abort = 0u;
    fence_barrier_init();
  }
  __syncthreads();
  pdl_begin();
  const int items = a.n_seqs * a.H, blocks = (a.dk + a.rows - 1) / a.rows;
  auto state_of = [&](int it, int b) {
    return a.state + (static_cast<size_t>(a.seq_slot[it / a.H]) * a.H + it % a.H) * static_cast<size_t>(a.dk) * a.dv +
           static_cast<size_t>(b) * a.rows * a.dv;
  };
  auto bytes_of = [&](int b) { return static_cast<uint32_t>(min(a.rows, a.dk - b * a.rows) * a.dv * 4); };
  int st = 0;
  uint32_t ph = 0;
  auto next = [&] {
    if (++st == LP_STAGES) {
      st = 0;
      ph ^= 1u;
    }
  };
  if (warp == LP_WORK / 32) {                                          // loader
    if (lane == 0) {
      bool ok = true;
      uint32_t asked = 0;
      for (int it = blockIdx.x; it < items && ok; it += gridDim.x) {
        if (a.q_len[it / a.H] <= 0) continue;
        for (int b = 0; b < blocks; ++b) {
          if (!(ok = ma_wait(&empty[st], ph ^ 1u, abort))) break;
          mbar_arrive_expect_tx(&full[st], bytes_of(b));
          bulk_load(ring + st * (LP_BYTES / 4), state_of(it, b), bytes_of(b), &full[st]);
          ++asked;
          next();
        }
      }
      if (!ok)                                                         // every copy that was asked for lands before the CTA leaves
        for (int s = 0; s < LP_STAGES; ++s)
          if (asked > static_cast<uint32_t>(s))
            for (uint32_t k = 0; k < (1u << 20) && !mbar_try_wait(&full[s], (asked - s - 1) / LP_STAGES & 1u); ++k) {}
    }
  } else if (warp > LP_WORK / 32) {                                    // storer
    if (lane == 0) {
      bool ok = true;
      for (int it = blockIdx.x; it < items && ok; it += gridDim.x) {
        if (a.q_len[it / a.H] <= 0) continue;
        for (int b = 0; b < blocks; ++b) {
          if (!(ok = ma_wait(&done[st], ph, abort))) break;
          asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(state_of(it, b)),
                       "r"(smem_u32(ring + st * (LP_BYTES / 4))), "r"(bytes_of(b))
                       : "memory");
          asm volatile("cp.async.bulk.commit_group;" ::: "memory");
          asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
          mbar_arrive(&empty[st]);
          next();
        }
      }
      asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    }
  } else {
    // inputs of an item: thread i holds channel i of q, k and v
    float nq = 0.f, nk = 0.f, nv = 0.f, nz = 0.f, nx = 0.f;
    auto fetch = [&](int it) {
      const int s = it / a.H, hd = it % a.H, hq = SSD ? hd / (a.H / a.G) : hd;
      const size_t t = static_cast<size_t>(a.q_start[s]);
      nq = tid < a.dk ? a.q[t * a.ld_q + hq * a.dk + tid] : 0.f;
      nk = tid < a.dk ? a.k[t * a.ld_k + hq * a.dk + tid] : 0.f;
      nv = tid < a.dv ? a.v[t * a.ld_v + hd * a.dv + tid] : 0.f;
      if (SSD) nx = a.step[t * a.ld_step + hd];
      else nz = tid < a.rdims ? a.tab[t * a.rdims + tid] : ((tid & 1) ? 0.f : 1.f);
    };
    auto keep = [&](int it, int buf) {
      const int hd = it % a.H;
      float* p = par + buf * 3 * 256;
      float d, b = 1.f;
      if (SSD) {
        b = softplus_(nx + a.bias[hd]);
        d = expf(-expf(a.hparam[hd]) * b);
      } else {
        d = a.hparam[hd];
        const float zo = __shfl_xor_sync(0xffffffffu, nz, 1), qo = __shfl_xor_sync(0xffffffffu, nq, 1), ko = __shfl_xor_sync(0xffffffffu, nk, 1);
        const bool odd = tid & 1;
        const float cs = odd ? zo : nz, sn = odd ? nz : -zo;
        nq = nq * cs + qo * sn;
        nk = nk * cs + ko * sn;
      }
      p[tid] = nk * b;
      p[256 + tid] = nq * a.qscale;
      p[512 + tid] = nv;
      if (tid == 0) sc[buf] = d;
    };
    auto meet = [] { asm volatile("bar.sync 1, 256;" ::: "memory"); };
    auto first_live = [&](int it) {
      while (it < items && a.q_len[it / a.H] <= 0) it += gridDim.x;
      return it;
    };
    const int c4 = a.dv / 4, RG = LP_WORK / c4, rg = tid / c4, cq = tid - rg * c4;
    int it = first_live(blockIdx.x), buf = 0;
    if (it < items) {
      fetch(it);
      keep(it, 0);
    }
    meet();
    bool ok = true;
    while (it < items) {                                               // (uniform over the eight warps; aborted or not, all meet)
      const int nx_it = first_live(it + gridDim.x);
      if (nx_it < items) fetch(nx_it);
      const int s = it / a.H;
      const bool fresh = a.kv_len[s] <= 1;                             // the first token of a sequence starts from zeros
      const float d = sc[buf];
      const float* p = par + buf * 3 * 256;
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f), v = o;
      if (rg < RG) v = *reinterpret_cast<const float4*>(p + 512 + 4 * cq);
      for (int b = 0; b < blocks; ++b) {
        ok = ok && __all_sync(0xffffffffu, ma_wait(&full[st], ph, abort));
        if (ok) {
          float4* S = reinterpret_cast<float4*>(ring + st * (LP_BYTES / 4));
          const int r0 = b * a.rows, nr = min(a.rows, a.dk - r0);
          if (rg < RG) {
#pragma unroll 4
            for (int r = rg; r < nr; r += RG) {
              float4 x = S[r * c4 + cq];
              if (fresh) x = make_float4(0.f, 0.f, 0.f, 0.f);
              const float kk = p[r0 + r], qq = p[256 + r0 + r];
              x = make_float4(d * x.x + kk * v.x, d * x.y + kk * v.y, d * x.z + kk * v.z, d * x.w + kk * v.w);
              o = make_float4(o.x + x.x * qq, o.y + x.y * qq, o.z + x.z * qq, o.w + x.w * qq);
              S[r * c4 + cq] = x;
            }
          }
          fence_proxy_async_smem();
          __syncwarp();
          if (lane == 0) mbar_arrive(&done[st]);
        }
        next();
      }
      if (nx_it < items) keep(nx_it, buf ^ 1);
      float* rd = red + buf * LP_WORK * 4;
      if (rg < RG) *reinterpret_cast<float4*>(rd + rg * a.dv + 4 * cq) = o;
      meet();
      if (tid < a.dv && ok) {
        float sum = 0.f;
        for (int g = 0; g < RG; ++g) sum += rd[g * a.dv + tid];
        a.out[static_cast<size_t>(a.q_start[s]) * a.ld_out + static_cast<size_t>(it % a.H) * a.dv + tid] = sum;
      }
      it = nx_it;
      buf ^= 1;
    }
    if (!ok && tid == 0) {
      if (g_abort_word != nullptr) *g_abort_word = 1u;
      atomicAdd(&g_step_gave_up, 1u);
    }
  }
  __syncthreads();                                                     // nobody leaves while copies of this CTA are in flight
}

}  // namespace

bool lin_chunk_supported(int dk, int dv) { return dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 256; }

int launch_lin_chunk(int ssd, const void* q, int ld_q, const void* k, int ld_k, const void* v, int ld_v, const float* step, int ld_step,
                     const float* bias, const float* hparam, float qscale, float* state, float* out, int ld_out, const int* q_start,
                     const int* q_len, const int* kv_len, const int* seq_slot, int n_seqs, int H, int G, int dk, int dv, cudaStream_t s) {
  if (n_seqs <= 0) return 0;
  auto al16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  if (!lin_chunk_supported(dk, dv) || G <= 0 || H % G != 0 || ld_q % 8 != 0 || ld_k % 8 != 0 || ld_v % 8 != 0 || ld_out % 4 != 0 || !al16(q) ||
      !al16(k) || !al16(v) || !al16(out))
    return -2;
  const ChunkArgs a{static_cast<const bf16*>(q), static_cast<const bf16*>(k), static_cast<const bf16*>(v), ld_q, ld_k, ld_v, step, ld_step,
                    bias, hparam, qscale, state, out, ld_out, q_start, q_len, kv_len, seq_slot, H, G, dk, dv};
#define B2B_LC(KT) return ssd ? launch_kt<KT, true>(a, n_seqs, s) : launch_kt<KT, false>(a, n_seqs, s)
  if (dk <= 64) B2B_LC(4);
  if (dk <= 128) B2B_LC(8);
  B2B_LC(16);
#undef B2B_LC
}

bool lin_step_supported(int n_seqs, int H, int dk, int dv) {
  return dk > 0 && dv > 0 && dv % 4 == 0 && dk <= 256 && dv <= 256 && static_cast<long long>(n_seqs) * H >= 148;
}

int launch_lin_step(int ssd, const float* q, int ld_q, const float* k, int ld_k, const float* v, int ld_v, const float* step, int ld_step,
                    const float* bias, const float* hparam, const float* tab, int rdims, float qscale, float* state, float* out, int ld_out,
                    const int* q_start, const int* q_len, const int* kv_len, const int* seq_slot, int n_seqs, int H, int G, int dk, int dv,
                    cudaStream_t s) {
  if (n_seqs <= 0) return 0;
  if (dk <= 0 || dv <= 0 || dv % 4 != 0 || dk > 256 || dv > 256 || G <= 0 || H % G != 0 || rdims < 0 || rdims > dk || rdims % 2 != 0 ||
      reinterpret_cast<uintptr_t>(state) % 16 != 0)
    return -2;
  const int per = LP_BYTES / (dv * 4);                                 // rows of a block; equal shares when a state needs several
  const int blocks = (dk + per - 1) / per, rows = (dk + blocks - 1) / blocks;
  const StepArgs a{q, k, v, ld_q, ld_k, ld_v, step, ld_step, bias, hparam, tab, rdims, qscale, state, out, ld_out, q_start, q_len, kv_len,
                   seq_slot, n_seqs, H, G, dk, dv, rows};
  constexpr size_t bytes = LP_STAGES * LP_BYTES + (2 * 3 * 256 + 4 + 2 * LP_WORK * 4) * 4 + 3 * LP_STAGES * 8 + 16;
  static bool set[2][64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 64 || !set[ssd != 0][dev]) {
    const cudaError_t e = ssd ? cudaFuncSetAttribute(lin_step_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes))
                              : cudaFuncSetAttribute(lin_step_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes));
    if (e != cudaSuccess) return static_cast<int>(e);
    if (dev < 64) set[ssd != 0][dev] = true;
  }
  const int items = n_seqs * H;
  const dim3 grid(items < 2 * 148 ? items : 2 * 148);
  return static_cast<int>(ssd ? launch_kernel(lin_step_kernel<true>, grid, dim3(LP_THREADS), bytes, s, 1u, a)
                              : launch_kernel(lin_step_kernel<false>, grid, dim3(LP_THREADS), bytes, s, 1u, a));
}

unsigned lin_step_gave_up() {
  unsigned n = 0;
  return cudaMemcpyFromSymbol(&n, g_step_gave_up, sizeof(n)) == cudaSuccess ? n : ~0u;
}

int set_wait_policy_step(uint32_t* abort_word, unsigned long long limit_ns) {
  cudaError_t e = cudaMemcpyToSymbol(g_abort_word, &abort_word, sizeof(abort_word));
  if (e == cudaSuccess) e = cudaMemcpyToSymbol(g_wait_limit_ns, &limit_ns, sizeof(limit_ns));
  return static_cast<int>(e);
}

}  // namespace b2b
