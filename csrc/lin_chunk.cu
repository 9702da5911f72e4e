// Linear recurrences with ONE decay per head and token, over whole chunks of a span on tensor cores (bf16 serving mode; single tokens,
// short spans and the float32 mode walk token by token in lin_scan, seqmix.cu, on the same fp32 states):
//     S_t = d_t S_(t-1) + b_t k_t v_t^T,   o_t = qscale S_t^T q_t          (S [dk, dv] per head and sequence slot)
//   state-space   d_t = exp(-exp(A_h) b_t), b_t = softplus(x_t + bias_h)    (q / k of a group of heads)
//   retention     d_t = decay_h, b_t = 1
// With c_t = log d_1 + ... + log d_t inside a chunk of 64 tokens that starts from S_0:
//     o_t = qscale (exp(c_t) S_0^T q_t + sum_(s <= t) exp(c_t - c_s) b_s (q_t . k_s) v_s)
//     S_L = exp(c_L) S_0 + sum_s exp(c_L - c_s) b_s k_s v_s^T
// so a chunk is four matrix products instead of 64 dependent steps.  q, k and v are bf16 (projections and convolved activations);
// everything that enters the recurrence besides them keeps fp32 precision: decays, their logarithms and sums, step sizes, the
// state (fp32 accumulators that stay in registers from chunk to chunk), and where a product of such numbers is an operand (weighted
// scores, weighted keys, the state in front of q) it is split into a high and a low bf16 part, 16 bits of mantissa together.
// A block = 32 state columns of one (sequence, head), eight warps.  Tokens of the chunk are the M dimension of the output products
// (four tiles of 16, two warps each that split the keys and the state rows); state rows are the M dimension of the update.
// The next chunk's rows come in by cp.async meanwhile.
// This translation unit is compiled WITHOUT --use_fast_math (exact expf / logf / softplus).
#include "kernels.h"

#include <cuda_bf16.h>

#include <cstdint>

#include "launch.cuh"

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

constexpr int LC_L = 64, LC_VB = 32, LC_THREADS = 256;
constexpr int LC_VS = LC_VB + 8;                       // row stride of value and state tiles (elements)

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
__global__ void __launch_bounds__(LC_THREADS)
    lin_chunk_kernel(const ChunkArgs a) {
  pdl_begin();
  constexpr int NP = 16 * KT, RS = NP + 8;             // row stride of q / k tiles
  constexpr int MT = KT > 8 ? KT / 8 : 1;              // state row tiles per warp (KT < 8: the last warps have none)
  constexpr int TILE = LC_L * RS, VT = LC_L * LC_VS;
  extern __shared__ __align__(16) uint8_t smem_[];
  bf16* qs = reinterpret_cast<bf16*>(smem_);           // [2][64][RS]
  bf16* ks = qs + 2 * TILE;
  bf16* vs = ks + 2 * TILE;                            // [2][64][VS]
  bf16* sh = vs + 2 * VT;                              // [NP][VS] state, high parts
  bf16* sl = sh + NP * LC_VS;
  float* ox = reinterpret_cast<float*>(sl + NP * LC_VS);      // [64][33] partial outputs of the second warp of a token tile
  float* cum = ox + LC_L * (LC_VB + 1);                // [64] c_t
  float* wst = cum + LC_L;                             // [64] b_s
  float* wup = wst + LC_L;                             // [64] exp(c_L - c_s) b_s
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

  // state rows of this warp: (warp * MT + m) * 16 + gid (+ 8), columns nt * 8 + 2 tig (+ 1)
  const bool owner = warp * MT < KT;
  float S[MT][4][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (warp * MT + m) * 16 + gid + (e >> 1) * 8, c = nt * 8 + 2 * tig + (e & 1);
        S[m][nt][e] = (owner && pos0 > 0 && r < a.dk && v0 + c < a.dv) ? Sg[static_cast<size_t>(r) * a.dv + c] : 0.f;
      }
  const float rate = SSD ? expf(a.hparam[hd]) : 0.f, bias = SSD ? a.bias[hd] : 0.f;
  const float logd = SSD ? 0.f : fmaxf(logf(a.hparam[hd]), -80.f);      // (a decay of zero: exp(-80) is zero beside any other term)

  auto stage = [&](int ch) {
    const int buf = ch & 1, tb = ch * LC_L;
    const int cols = a.dk / 8;
    for (int e = tid; e < LC_L * (NP / 8); e += LC_THREADS) {
      const int r = e / (NP / 8), c = e % (NP / 8);
      const bool ok = tb + r < n && c < cols;
      const size_t t = static_cast<size_t>(t0 + (ok ? tb + r : 0));
      cp16(sptr(qs + buf * TILE + r * RS + c * 8), qg + t * a.ld_q + (ok ? c * 8 : 0), ok);
      cp16(sptr(ks + buf * TILE + r * RS + c * 8), kg + t * a.ld_k + (ok ? c * 8 : 0), ok);
    }
    {
      const int r = tid >> 2, c = tid & 3;             // 64 rows x 4 pieces of 8 columns
      const bool ok = tb + r < n && v0 + c * 8 < a.dv;
      const size_t t = static_cast<size_t>(t0 + (ok ? tb + r : 0));
      cp16(sptr(vs + buf * VT + r * LC_VS + c * 8), vg + t * a.ld_v + (ok ? c * 8 : 0), ok);
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  // step size of token tid of a chunk (threads 0 .. 63), read a chunk ahead
  auto load_step = [&](int ch) {
    const int i = ch * LC_L + tid;
    return (SSD && tid < LC_L && i < n) ? a.step[static_cast<size_t>(t0 + i) * a.ld_step + hd] : 0.f;
  };

  const int nch = (n + LC_L - 1) / LC_L;
  stage(0);
  float xs = load_step(0);
  const int mt = warp & 3, kh = warp >> 2;             // token tile; which half of the keys / of the state rows
  for (int ch = 0; ch < nch; ++ch) {
    const int buf = ch & 1, tb = ch * LC_L;
    if (ch + 1 < nch) stage(ch + 1);
    else asm volatile("cp.async.commit_group;\n" ::: "memory");
    // logarithms of the decays, their running sums (two warps, then the second adds the first one's total)
    if (tid < LC_L) {
      const bool in = tb + tid < n;
      float b = in ? 1.f : 0.f, lg = in ? logd : 0.f;
      if (SSD) {
        b = in ? softplus_(xs + bias) : 0.f;
        lg = -rate * b;
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float u = __shfl_up_sync(0xffffffffu, lg, o);
        if (lane >= o) lg += u;
      }
      cum[tid] = lg;
      wst[tid] = b;
    }
    if (ch + 1 < nch) xs = load_step(ch + 1);
    // the state in front of this chunk as an operand
    if (owner) {
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int r = (warp * MT + m) * 16 + gid + e * 8, c = nt * 8 + 2 * tig;
            uint32_t hi, lo;
            split2(S[m][nt][2 * e], S[m][nt][2 * e + 1], &hi, &lo);
            *reinterpret_cast<uint32_t*>(sh + r * LC_VS + c) = hi;
            *reinterpret_cast<uint32_t*>(sl + r * LC_VS + c) = lo;
          }
    }
    asm volatile("cp.async.wait_group 1;\n" ::: "memory");
    __syncthreads();
    if (tid >= 32 && tid < LC_L) cum[tid] += cum[31];
    __syncthreads();
    if (tid < LC_L) wup[tid] = expf(cum[LC_L - 1] - cum[tid]) * wst[tid];
    const float clast = cum[LC_L - 1];

    // ---- outputs of 16 tokens against half of the keys and half of the state rows
    float op[4][4], os[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) op[i][e] = os[i][e] = 0.f;
    const int r0 = mt * 16 + gid, r1 = r0 + 8;
    const float cr0 = cum[r0], cr1 = cum[r1];
    const uint32_t qa = sptr(qs + buf * TILE + (mt * 16 + (lane & 15)) * RS + (lane >> 4) * 8);
    const uint32_t vt_off = (((lane & 7) + ((lane >> 3) & 1) * 8) * LC_VS + (lane >> 4) * 8) * 2;
    if (kh * 32 <= mt * 16 + 15) {                     // (keys behind every token of the tile: nothing)
      float g[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) g[i][e] = 0.f;
      const uint32_t kb = sptr(ks + buf * TILE + (kh * 32 + (lane & 7) + (lane >> 4) * 8) * RS + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int kk = 0; kk < KT; ++kk) {
        uint32_t af[4], b0[4], b1[4];
        ldsm(af, qa + kk * 32);
        ldsm(b0, kb + kk * 32);
        ldsm(b1, kb + (16 * RS + kk * 16) * 2);
        mma(g[0], af, b0[0], b0[1]);
        mma(g[1], af, b0[2], b0[3]);
        mma(g[2], af, b1[0], b1[1]);
        mma(g[3], af, b1[2], b1[3]);
      }
#pragma unroll
      for (int k2 = 0; k2 < 2; ++k2) {                 // 16 keys: weighted scores -> A operand (high, low), times the values
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int nt = 2 * k2 + h, c = kh * 32 + nt * 8 + 2 * tig;
          const float ca = cum[c], cb = cum[c + 1], wa = wst[c], wb = wst[c + 1];
          const float p00 = c <= r0 ? g[nt][0] * expf(cr0 - ca) * wa : 0.f, p01 = c + 1 <= r0 ? g[nt][1] * expf(cr0 - cb) * wb : 0.f;
          const float p10 = c <= r1 ? g[nt][2] * expf(cr1 - ca) * wa : 0.f, p11 = c + 1 <= r1 ? g[nt][3] * expf(cr1 - cb) * wb : 0.f;
          split2(p00, p01, &ph[2 * h], &pl[2 * h]);
          split2(p10, p11, &ph[2 * h + 1], &pl[2 * h + 1]);
        }
        const uint32_t va = sptr(vs + buf * VT + (kh * 32 + k2 * 16) * LC_VS) + vt_off;
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
    }
    {
      const uint32_t ha = sptr(sh) + vt_off, la = sptr(sl) + vt_off;
#pragma unroll
      for (int k2 = 0; k2 < KT / 2; ++k2) {
        const int kk = kh * (KT / 2) + k2;
        uint32_t af[4];
        ldsm(af, qa + kk * 32);
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
    {
      const float e0 = expf(cr0), e1 = expf(cr1);
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        op[nt][0] += e0 * os[nt][0];
        op[nt][1] += e0 * os[nt][1];
        op[nt][2] += e1 * os[nt][2];
        op[nt][3] += e1 * os[nt][3];
      }
      if (kh == 1) {
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) ox[(mt * 16 + gid + (e >> 1) * 8) * (LC_VB + 1) + nt * 8 + 2 * tig + (e & 1)] = op[nt][e];
      }
    }
    __syncthreads();                                   // partial outputs and update weights are there

    // ---- state behind this chunk: rows of the warp's tiles over all tokens
    if (owner) {
      const float dec = expf(clast);
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[m][nt][e] *= dec;
#pragma unroll
      for (int k2 = 0; k2 < LC_L / 16; ++k2) {
        const int t = k2 * 16 + 2 * tig;
        const float w0 = wup[t], w1 = wup[t + 1], w8 = wup[t + 8], w9 = wup[t + 9];
        uint32_t b[2][4];
        const uint32_t va = sptr(vs + buf * VT + k2 * 16 * LC_VS) + vt_off;
        ldsm_t(b[0], va);
        ldsm_t(b[1], va + 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t kf[4], hi[4], lo[4];
          ldsm_t(kf, sptr(ks + buf * TILE + (k2 * 16 + (lane & 7) + (lane >> 4) * 8) * RS + (warp * MT + m) * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&kf[e]));
            split2(f.x * (e < 2 ? w0 : w8), f.y * (e < 2 ? w1 : w9), &hi[e], &lo[e]);
          }
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            mma(S[m][2 * j], hi, b[j][0], b[j][1]);
            mma(S[m][2 * j + 1], hi, b[j][2], b[j][3]);
            mma(S[m][2 * j], lo, b[j][0], b[j][1]);
            mma(S[m][2 * j + 1], lo, b[j][2], b[j][3]);
          }
        }
      }
    }
    if (kh == 0) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = mt * 16 + gid + e * 8;
        if (tb + r >= n) continue;
        float* dst = a.out + static_cast<size_t>(t0 + tb + r) * a.ld_out + static_cast<size_t>(hd) * a.dv + v0;
        const float* part = ox + r * (LC_VB + 1);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          const int c = nt * 8 + 2 * tig;
          if (v0 + c < a.dv)                           // (dv is a multiple of 8)
            *reinterpret_cast<float2*>(dst + c) = make_float2((op[nt][2 * e] + part[c]) * a.qscale, (op[nt][2 * e + 1] + part[c + 1]) * a.qscale);
        }
      }
    }
    __syncthreads();                                   // tiles, state operand and partial outputs may be written again
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (warp * MT + m) * 16 + gid + (e >> 1) * 8, c = nt * 8 + 2 * tig + (e & 1);
        if (owner && r < a.dk && v0 + c < a.dv) Sg[static_cast<size_t>(r) * a.dv + c] = S[m][nt][e];
      }
}

template <int KT, bool SSD>
int launch_kt(const ChunkArgs& a, int n_seqs, cudaStream_t s) {
  constexpr int NP = 16 * KT, RS = NP + 8;
  constexpr size_t bytes = static_cast<size_t>(4 * LC_L * RS + 2 * LC_L * LC_VS + 2 * NP * LC_VS) * 2 +
                           static_cast<size_t>(LC_L * (LC_VB + 1) + 3 * LC_L) * 4;
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

}  // namespace

bool lin_chunk_supported(int dk, int dv) { return dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 256; }

int launch_lin_chunk(int ssd, const void* q, int ld_q, const void* k, int ld_k, const void* v, int ld_v, const float* step, int ld_step,
                     const float* bias, const float* hparam, float qscale, float* state, float* out, int ld_out, const int* q_start,
                     const int* q_len, const int* kv_len, const int* seq_slot, int n_seqs, int H, int G, int dk, int dv, cudaStream_t s) {
  if (n_seqs <= 0) return 0;
  auto al16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  if (!lin_chunk_supported(dk, dv) || G <= 0 || H % G != 0 || ld_q % 8 != 0 || ld_k % 8 != 0 || ld_v % 8 != 0 || ld_out % 2 != 0 || !al16(q) ||
      !al16(k) || !al16(v) || reinterpret_cast<uintptr_t>(out) % 8 != 0)
    return -2;
  const ChunkArgs a{static_cast<const bf16*>(q), static_cast<const bf16*>(k), static_cast<const bf16*>(v), ld_q, ld_k, ld_v, step, ld_step,
                    bias, hparam, qscale, state, out, ld_out, q_start, q_len, kv_len, seq_slot, H, G, dk, dv};
#define B2B_LC(KT) return ssd ? launch_kt<KT, true>(a, n_seqs, s) : launch_kt<KT, false>(a, n_seqs, s)
  if (dk <= 64) B2B_LC(4);
  if (dk <= 128) B2B_LC(8);
  B2B_LC(16);
#undef B2B_LC
}

}  // namespace b2b
