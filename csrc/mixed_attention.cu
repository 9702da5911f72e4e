// Softmax attention with mixed heads over the paged KV cache, bf16 serving mode (the exact kernel of every mode is
// softmax_attention in seqmix.cu).  The scores of all heads are mixed by a learned matrix in front of the softmax; in
// absorbed form (talk_prep, seqmix.cu) head h has ONE query row over the whole cached key row of all key heads,
//     s[h, i, j] = qm[i, h, :] . krow[j, :] - slope_h (i - j)        (GD = key heads x channels products per score)
//     out[i, h, :] = sum_j softmax_j(s) krow[j, v0(h) : v0(h) + V]    (the keys are the values)
// over the keys j <= i, and j > i - window when window > 0; sink [H] (optional): exp(sink_h) joins the denominator.
//
//   * mixed_attention_tc_kernel   spans: tcgen05.mma, 128 queries of one head per CTA, scores and output in tensor memory,
//                                 key tiles of 128 rows streamed by TMA in slabs of 64 channels through a ring; the slabs
//                                 that hold the head's values come a second time (from L2) for the second product, so no
//                                 slab outlives the MMAs that follow it.  Warp roles: 0 TMA producer, 1 MMA issuer, 2..9
//                                 softmax (two threads per query, 64 keys of a tile each).
//   * mixed_attention_dec_kernel  single decoded tokens (and spans of two): a cluster of CTAs shares the keys of one query,
//                                 heads are the N dimension of mma.sync (keys, then channels are the M dimension), key
//                                 tiles are staged once for all heads with cp.async; partial results merge through
//                                 distributed shared memory.
// Scores, bias, masks, running maximum and sums are fp32; P is rounded to bf16 as the operand of the second product.
// This translation unit is compiled WITHOUT --use_fast_math; the exponentials are the hardware exp2 (2^-22 relative).
#include "kernels.h"

#include <cuda.h>

#include "common.cuh"
#include "launch.cuh"
#include "tmem.cuh"

namespace b2b {

int make_tmap_shared(CUtensorMap* m, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows,
                     int elt_bytes);

namespace {

typedef __nv_bfloat16 bf16;
constexpr float MA_LOG2E = 1.4426950408889634f;
constexpr int MA_PAGE = 64;

struct MixedArgs {
  bf16* out;
  const int* block_table;
  const int* q_start;
  const int* q_len;
  const int* kv_len;
  const float* slope;      // [H] or null
  const float* sink;       // [H] or null
  int ld_out, max_pages, H, Gv, GD, V, window;
  int ns, nst;             // slabs of 64 channels per key row, stages of the ring
};

__device__ unsigned int g_mixed_gave_up = 0;          // CTAs whose waits ran out since the module was loaded

// ------------------------------------------------------------------------------------------------ spans (tcgen05)
constexpr int MT_THREADS = 320, MT_BKV = 128, MT_SLAB = 128 * 128;      // a slab: 128 rows x 64 channels
constexpr int MT_MAX_STAGES = 13;
constexpr int MT_SMEM_MAX = 227 * 1024;
constexpr int MT_BAR_BYTES = 512 + 2048;      // barriers, row maxima of the two halves (double-buffered)

// QRES: the query tile (128 rows x GD channels) stays in shared memory; otherwise its slabs travel with the key slabs
template <bool QRES>
__global__ void __launch_bounds__(MT_THREADS, 1)
    mixed_attention_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                              const MixedArgs p) {
  constexpr uint32_t S_COL = 0, O_COL = 2 * MT_BKV, TCOLS = 512;
  constexpr int STAGE = QRES ? MT_SLAB : 2 * MT_SLAB;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* q_s = smem;                                            // QRES: [ns][MT_SLAB]
  uint8_t* ring = smem + (QRES ? p.ns * MT_SLAB : 0);             // [nst][STAGE]: key slab (| query slab)
  uint64_t* bars = reinterpret_cast<uint64_t*>(ring + p.nst * STAGE);
  uint64_t* full = bars;
  uint64_t* empty = bars + MT_MAX_STAGES;
  uint64_t* s_full = bars + 2 * MT_MAX_STAGES;
  uint64_t* p_ready = s_full + 2;
  uint64_t* pv_done = s_full + 3;
  uint64_t* q_full = s_full + 4;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(s_full + 5);
  float* half_s = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(bars) + 512);      // [2 tiles][2 halves][128]
  volatile uint32_t* abort = tmem_slot + 1;
  volatile uint32_t* issued = tmem_slot + 2;                      // slabs the producer has asked for

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < p.nst; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    mbar_init(p_ready, 8);
    mbar_init(pv_done, 1);
    mbar_init(q_full, 1);
    *abort = 0u;
    *issued = 0u;
    fence_barrier_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_k);
  }
  if (warp == 1) tmem_alloc<TCOLS>(tmem_slot);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  pdl_launch_dependents();                                        // (every CTA of the grid owns its tensor memory by then)
  pdl_wait();

  const int seq = blockIdx.z, hd = blockIdx.y;
  const int qlen = p.q_len[seq], kvlen = p.kv_len[seq];
  const int q0 = blockIdx.x * 128;
  const bool active = q0 < qlen;                                  // CTA-uniform
  const int nq = min(128, qlen - q0);
  const int qtok0 = p.q_start[seq] + q0;
  const int pos0 = kvlen - qlen + q0;                             // position of the block's first query
  const int kv_hi = pos0 + nq;
  const int kv_lo = p.window > 0 ? max(0, pos0 - p.window + 1) : 0;
  const int t_lo = kv_lo / MT_BKV;
  const int nt = active ? (kv_hi + MT_BKV - 1) / MT_BKV - t_lo : 0;
  const int gv = hd / (p.H / p.Gv);
  const int v0 = gv * p.V / 64;                                   // first slab and number of slabs with the head's values
  const int nv = (gv * p.V + p.V - 1) / 64 - v0 + 1;

  if (!active) {
  } else if (warp == 0) {
    if (elect_one()) {
      if (QRES) {
        mbar_arrive_expect_tx(q_full, p.ns * MT_SLAB);
        for (int c = 0; c < p.ns; ++c) tma_load_2d(q_s + c * MT_SLAB, &tm_q, q_full, hd * p.GD + c * 64, qtok0);
      }
      const int* bt = p.block_table + static_cast<size_t>(seq) * p.max_pages;
      int st = 0;
      uint32_t ph = 0, g = 0;
      // the slabs c0 .. c0 + cn - 1 of key tile n, for the first product (with the query slabs when they travel) or the second
      auto tile = [&](int n, int c0, int cn, bool with_q) {
        const int pg = 2 * (t_lo + n);
        const int page0 = bt[pg];
        const int page1 = (pg + 1 < p.max_pages && (pg + 1) * MA_PAGE < kv_hi) ? bt[pg + 1] : page0;   // past the newest key: any rows
        for (int c = c0; c < c0 + cn; ++c) {
          if (!ma_wait(&empty[st], ph ^ 1u, abort)) return false;
          uint8_t* dst = ring + st * STAGE;
          mbar_arrive_expect_tx(&full[st], with_q ? 2 * MT_SLAB : MT_SLAB);
          tma_load_2d(dst, &tm_k, &full[st], c * 64, page0 * MA_PAGE);
          tma_load_2d(dst + MT_SLAB / 2, &tm_k, &full[st], c * 64, page1 * MA_PAGE);
          if (with_q) tma_load_2d(dst + MT_SLAB, &tm_q, &full[st], hd * p.GD + c * 64, qtok0);
          *issued = ++g;
          if (++st == p.nst) {
            st = 0;
            ph ^= 1u;
          }
        }
        return true;
      };
      bool ok = tile(0, 0, p.ns, !QRES);
      for (int n = 0; n < nt && ok; ++n) {                        // the order in which the MMA warp consumes
        if (n + 1 < nt) ok = tile(n + 1, 0, p.ns, !QRES);
        ok = ok && tile(n, v0, nv, false);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    constexpr uint32_t idesc_s = make_idesc_bf16(128, MT_BKV);
    constexpr uint32_t idesc_o = make_idesc_bf16(128, 64) | (1u << 16);      // B operand (values) is MN-major
    int st = 0;
    uint32_t ph = 0;
    auto all = [&](bool b) { return __all_sync(0xffffffffu, b) != 0; };
    auto next = [&] {
      if (++st == p.nst) {
        st = 0;
        ph ^= 1u;
      }
    };
    auto qk = [&](int n) {
      const uint32_t d = tmem + S_COL + static_cast<uint32_t>(n & 1) * MT_BKV;
      for (int i = 0; i < p.ns; ++i) {
        if (!all(ma_wait(&full[st], ph, abort))) return false;
        tc_fence_after();
        if (elect_one()) {
          const uint8_t* ks = ring + st * STAGE;
          const uint8_t* qs = QRES ? q_s + i * MT_SLAB : ks + MT_SLAB;
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            umma_bf16(d, make_sw128_kmajor_desc(smem_u32(qs)) + static_cast<uint64_t>(kk * 2),
                      make_sw128_kmajor_desc(smem_u32(ks)) + static_cast<uint64_t>(kk * 2), idesc_s, (i > 0 || kk > 0) ? 1u : 0u);
          umma_commit(&empty[st]);
          if (i == p.ns - 1) umma_commit(&s_full[n & 1]);
        }
        __syncwarp();
        next();
      }
      return true;
    };
    bool ok = !QRES || all(ma_wait(q_full, 0, abort));
    ok = ok && qk(0);
    for (int n = 0; n < nt && ok; ++n) {
      if (n + 1 < nt && !(ok = qk(n + 1))) break;                // next scores run while this tile's softmax does
      if (!(ok = all(ma_wait(p_ready, static_cast<uint32_t>(n & 1), abort)))) break;
      for (int j = 0; j < nv; ++j) {
        if (!(ok = all(ma_wait(&full[st], ph, abort)))) break;
        tc_fence_after();
        if (elect_one()) {
          const uint32_t vb = smem_u32(ring + st * STAGE);
#pragma unroll
          for (int kk = 0; kk < MT_BKV / 16; ++kk)
            ma_mma_ts(tmem + O_COL + j * 64, tmem + S_COL + static_cast<uint32_t>(n & 1) * MT_BKV + kk * 8,
                      ma_value_desc(vb + kk * (16 * 128)), idesc_o, (n > 0 || kk > 0) ? 1u : 0u);
          umma_commit(&empty[st]);
          if (j == nv - 1) umma_commit(pv_done);
        }
        __syncwarp();
        next();
      }
    }
  } else {
    const int quarter = warp & 3, half = (warp - 2) >> 2;         // half: which 64 keys of a tile this warp has
    const int i = quarter * 32 + lane;                            // query of the block
    const bool row_valid = i < nq;
    const int qpos = pos0 + i;
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(quarter * 32) << 16);
    const float sl = p.slope != nullptr ? p.slope[hd] * MA_LOG2E : 0.f;
    float m_ref = p.sink != nullptr ? p.sink[hd] * MA_LOG2E : -INFINITY, l = p.sink != nullptr && half == 0 ? 1.f : 0.f;
    auto all = [&](bool b) { return __all_sync(0xffffffffu, b) != 0; };
    // the two threads of a query exchange a number; every softmax warp takes part nt + 1 times, aborted or not
    auto meet = [] { asm volatile("bar.sync 1, 256;" ::: "memory"); };
    constexpr int NE = MT_BKV / 2;

    auto tile = [&](int n, auto masked) {
      const int kb = (t_lo + n) * MT_BKV + half * NE, b = n & 1;
      if (!all(ma_wait(&s_full[b], static_cast<uint32_t>((n >> 1) & 1), abort))) {
        meet();
        return false;
      }
      tc_fence_after();
      const uint32_t s_addr = lane_addr + S_COL + static_cast<uint32_t>(b) * MT_BKV;
      uint32_t r[NE];
#pragma unroll
      for (int c = 0; c < NE; c += 32) ma_ld32(s_addr + half * NE + c, r + c);
#pragma unroll
      for (int c = 0; c < NE; c += 32) ma_ld_fence(r + c);
      const float nb = -sl * static_cast<float>(qpos - kb);
      float mrow = -INFINITY;
#pragma unroll
      for (int e = 0; e < NE; ++e) {
        float sc = __fmaf_rn(__uint_as_float(r[e]), MA_LOG2E, __fmaf_rn(sl, static_cast<float>(e), nb));
        if constexpr (decltype(masked)::value) {
          const int j = kb + e;
          const bool ok = row_valid && j <= qpos && (p.window <= 0 || j > qpos - p.window);
          sc = ok ? sc : -INFINITY;
        }
        r[e] = __float_as_uint(sc);
        mrow = fmaxf(mrow, sc);
      }
      float* hs = half_s + (n & 1) * 256 + i;
      hs[half * 128] = mrow;
      tc_fence_before();                                          // (both halves have read their scores before P goes over them)
      meet();
      tc_fence_after();
      mrow = fmaxf(mrow, hs[(half ^ 1) * 128]);
      // lazy rescaling: the reference stays while the new maximum is within 2^8 of it
      float alpha = 1.f;
      if (mrow > m_ref + 8.f || (m_ref == -INFINITY && mrow > -INFINITY)) {
        alpha = (m_ref == -INFINITY) ? 0.f : ex2(m_ref - mrow);
        m_ref = mrow;
      }
      const float mr = (m_ref == -INFINITY) ? 0.f : m_ref;        // nothing visible so far: exp2(-inf) = 0
      float lsum = 0.f;
      {
        uint32_t pk[32];
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          const float p0 = ex2(__uint_as_float(r[2 * j]) - mr);
          const float p1 = ex2(__uint_as_float(r[2 * j + 1]) - mr);
          lsum += p0 + p1;
          pk[j] = pack2(p0, p1);
        }
        ma_st32(s_addr + half * 32, pk);                          // over the scores of this tile, which are in registers
      }
      if (n > 0) {
        if (!all(ma_wait(pv_done, static_cast<uint32_t>((n - 1) & 1), abort))) return false;
        tc_fence_after();
        if (__any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll 1
          for (int c = half * 32; c < nv * 64; c += 64) {
            uint32_t o[32];
            ma_ld32(lane_addr + O_COL + c, o);
            ma_ld_fence(o);
#pragma unroll
            for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * alpha);
            ma_st32(lane_addr + O_COL + c, o);
          }
        }
      }
      ma_st_wait();
      l = l * alpha + lsum;
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
      return true;
    };

    bool ok = true;
    for (int n = 0; n < nt; ++n) {
      if (!ok) {
        meet();
        continue;
      }
      const int kb = (t_lo + n) * MT_BKV;
      const bool every = nq == 128 && kb + MT_BKV - 1 <= pos0 && (p.window <= 0 || kb > pos0 + nq - 1 - p.window);
      ok = every ? tile(n, std::false_type{}) : tile(n, std::true_type{});
    }
    half_s[(nt & 1) * 256 + half * 128 + i] = l;
    meet();
    l += half_s[(nt & 1) * 256 + (half ^ 1) * 128 + i];
    if (ok) ok = all(ma_wait(pv_done, static_cast<uint32_t>((nt - 1) & 1), abort));
    if (ok) {
      tc_fence_after();
      const float inv = l > 0.f ? 1.f / l : 0.f;
      const int off = gv * p.V - v0 * 64;
      bf16* dst = p.out + static_cast<size_t>(qtok0 + i) * p.ld_out + hd * p.V;
#pragma unroll 1
      for (int c = half * 32; c < p.V; c += 64) {
        uint32_t o[32];
        ma_ld32(lane_addr + O_COL + off + c, o);
        ma_ld_fence(o);
        if (!row_valid) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (c + 8 * j >= p.V) break;
          uint32_t w[4];
#pragma unroll
          for (int e = 0; e < 4; ++e)
            w[e] = pack2(__uint_as_float(o[8 * j + 2 * e]) * inv, __uint_as_float(o[8 * j + 2 * e + 1]) * inv);
          *reinterpret_cast<uint4*>(dst + c + 8 * j) = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (active && *abort != 0u) {
    // a wait ran out: report it, let the copies that are still in flight land (again bounded), leave
    if (threadIdx.x == 0) {
      if (g_abort_word != nullptr) *g_abort_word = 1u;
      atomicAdd(&g_mixed_gave_up, 1u);
      const uint32_t g = *issued;
      for (int s = 0; s < p.nst; ++s) {
        if (g <= static_cast<uint32_t>(s)) break;
        const uint32_t uses = (g - s - 1) / p.nst;                // the stage's last phase
        for (uint32_t k = 0; k < (1u << 20) && !mbar_try_wait(&full[s], uses & 1u); ++k) {}
      }
      if (QRES)
        for (uint32_t k = 0; k < (1u << 20) && !mbar_try_wait(q_full, 0); ++k) {}
    }
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc<TCOLS>(tmem);
  }
}

// ------------------------------------------------------------------------------------------------ decode (mma.sync)
__device__ __forceinline__ void md_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void md_ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void md_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void md_cp16(uint32_t dst, const void* src, bool take) {      // !take: zeros
  const int n = take ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void md_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void md_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }
__device__ __forceinline__ float md_ld_cluster(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}

constexpr int MD_WARPS = 8, MD_THREADS = 32 * MD_WARPS;
constexpr int MD_MAX_HEADS = 64;
__host__ __device__ constexpr int md_row(int GD) { return (GD + 15) / 16 * 16 + 8; }     // elements; 16-byte chunks per row are odd
struct MdLayout {
  int qs, ks, ps, part, red, out, bytes;          // byte offsets
};
__host__ __device__ inline MdLayout md_layout(int H, int hp16, int Gv, int GD, int V, int KT) {
  const int rs = md_row(GD) * 2, per8 = (H / Gv + 7) / 8 * 8, ksp = MD_WARPS / (KT / 16);
  MdLayout L;
  L.qs = 0;
  L.ks = L.qs + hp16 * 16 * rs;
  L.ps = L.ks + 2 * KT * rs;
  L.part = L.ps + Gv * per8 * (KT + 8) * 2;
  L.red = L.part + ksp * hp16 * 16 * (KT + 4) * 4;
  L.bytes = L.red + 3 * MD_MAX_HEADS * 4;         // alpha, maximum, sum per head
  L.out = L.ks;                                   // the outputs take the place of the key tiles at the end
  if (H * V * 4 > 2 * KT * rs) {
    L.out = L.bytes;
    L.bytes += H * V * 4;
  }
  return L;
}

// grid (queries of a span, sequences, splits), cluster (1, 1, splits).  HP16: heads in units of 16 (zero rows behind the
// last); KT: keys per tile; MU: output tiles (16 channels x 8 heads of one value head) per warp.
template <int HP16, int KT, int MU>
__global__ void __launch_bounds__(MD_THREADS)
    mixed_attention_dec_kernel(const bf16* __restrict__ q, const bf16* __restrict__ kc, const MixedArgs p) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int MT = KT / 16, KSP = MD_WARPS / MT;                // key tiles of 16 rows; the channels are split KSP ways
  extern __shared__ __align__(128) uint8_t smem[];
  const MdLayout L = md_layout(p.H, HP16, p.Gv, p.GD, p.V, KT);
  const int rs = md_row(p.GD), hp = p.H / p.Gv, per8 = (hp + 7) / 8 * 8;
  bf16* ps = reinterpret_cast<bf16*>(smem + L.ps);                // [Gv * per8][KT + 8]
  float* part = reinterpret_cast<float*>(smem + L.part);          // [KSP][HP16 * 16][KT + 4]
  float* red = reinterpret_cast<float*>(smem + L.red);            // alpha [64], maximum [64], sum [64]
  float* outp = reinterpret_cast<float*>(smem + L.out);           // [H][V]
  const uint32_t qs_a = smem_u32(smem + L.qs), ks_a = smem_u32(smem + L.ks), ps_a = smem_u32(smem + L.ps);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int seq = blockIdx.y, i = blockIdx.x, splits = gridDim.z, split = blockIdx.z;
  const int qlen = p.q_len[seq];
  if (i >= qlen) return;                                          // the whole cluster leaves
  const int t = p.q_start[seq] + i, pi = p.kv_len[seq] - qlen + i;
  const int lo = p.window > 0 ? max(0, pi - p.window + 1) : 0;
  const int first = lo / KT, n_all = pi / KT - first + 1, each = (n_all + splits - 1) / splits;
  const int tb = first + min(n_all, split * each), te = first + min(n_all, (split + 1) * each);
  const int* bt = p.block_table + static_cast<size_t>(seq) * p.max_pages;

  // padding that no copy writes: channels GD .. of every row (query rows, both key buffers), query rows and P rows of no head
  {
    const uint4 z = make_uint4(0u, 0u, 0u, 0u);
    const int tail = rs - p.GD;                                   // 8 or 16 elements
    for (int e = threadIdx.x; e < (HP16 * 16 + 2 * KT) * (tail / 8); e += MD_THREADS) {
      const int r = e / (tail / 8), c = e % (tail / 8);
      *reinterpret_cast<uint4*>(smem + (static_cast<size_t>(r) * rs + p.GD + c * 8) * 2) = z;
    }
    for (int e = threadIdx.x; e < (HP16 * 16 - p.H) * (p.GD / 8); e += MD_THREADS)
      *reinterpret_cast<uint4*>(smem + (static_cast<size_t>(p.H + e / (p.GD / 8)) * rs + e % (p.GD / 8) * 8) * 2) = z;
    for (int e = threadIdx.x; e < p.Gv * per8 * (KT + 8) / 8; e += MD_THREADS) reinterpret_cast<uint4*>(ps)[e] = z;
  }
  const int c8 = p.GD / 8;
  {
    const bf16* qr = q + static_cast<size_t>(t) * p.H * p.GD;
    for (int e = threadIdx.x; e < p.H * c8; e += MD_THREADS)
      md_cp16(qs_a + (e / c8 * rs + e % c8 * 8) * 2, qr + static_cast<size_t>(e) * 8, true);
  }
  auto stage = [&](int tl) {
    const int kb = tl * KT;
    const size_t base = static_cast<size_t>(bt[kb >> 6]) * MA_PAGE + (kb & 63);          // a tile lies inside one page
    const uint32_t dst = ks_a + (tl & 1) * KT * rs * 2;
    for (int e = threadIdx.x; e < KT * c8; e += MD_THREADS) {
      const int r = e / c8, c = e - r * c8, j = kb + r;
      md_cp16(dst + (r * rs + c * 8) * 2, kc + (base + r) * p.GD + c * 8, j >= lo && j <= pi);
    }
  };
  if (tb < te) stage(tb);
  md_commit();

  float m_[HP16 * 2], l_[HP16 * 2];                               // of heads warp, warp + 8, ... (the same in every lane)
#pragma unroll
  for (int k = 0; k < HP16 * 2; ++k) {
    const int h = warp + 8 * k;
    const bool has = split == 0 && p.sink != nullptr && h < p.H;
    m_[k] = has ? p.sink[h] * MA_LOG2E : -INFINITY;
    l_[k] = has ? 1.f : 0.f;
  }
  float o[MU][4];
#pragma unroll
  for (int u = 0; u < MU; ++u) o[u][0] = o[u][1] = o[u][2] = o[u][3] = 0.f;
  const int mtv = (p.V + 15) / 16, ntg = per8 / 8, units = p.Gv * mtv * ntg;
  const int mt = warp % MT, kp = warp / MT;
  const int k16 = (p.GD + 15) / 16, kper = (k16 + KSP - 1) / KSP;
  const int kbeg = min(k16, kp * kper), kend = min(k16, kbeg + kper);

  for (int tl = tb; tl < te; ++tl) {
    if (tl + 1 < te) stage(tl + 1);
    md_commit();
    md_wait<1>();
    __syncthreads();                                              // this tile is staged (and the last one's partials are read)
    const uint32_t kt_a = ks_a + (tl & 1) * KT * rs * 2;
    {
      float acc[HP16 * 2][4];
#pragma unroll
      for (int n = 0; n < HP16 * 2; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
      const uint32_t aa = kt_a + ((mt * 16 + (lane & 15)) * rs + (lane >> 4) * 8) * 2;
      const uint32_t ba = qs_a + (((lane & 7) + (lane >> 4) * 8) * rs + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll 4
      for (int k = kbeg; k < kend; ++k) {
        uint32_t a[4];
        md_ldsm(a, aa + k * 32);
#pragma unroll
        for (int n = 0; n < HP16; ++n) {
          uint32_t b[4];
          md_ldsm(b, ba + (n * 16 * rs + k * 16) * 2);
          md_mma(acc[2 * n], a, b[0], b[1]);
          md_mma(acc[2 * n + 1], a, b[2], b[3]);
        }
      }
      float* pp = part + static_cast<size_t>(kp) * HP16 * 16 * (KT + 4) + mt * 16 + gid;
#pragma unroll
      for (int n = 0; n < HP16 * 2; ++n) {
        float* c = pp + (n * 8 + 2 * tig) * (KT + 4);
        c[0] = acc[n][0];
        c[KT + 4] = acc[n][1];
        c[8] = acc[n][2];
        c[KT + 4 + 8] = acc[n][3];
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < HP16 * 2; ++k) {
      const int h = warp + 8 * k;
      if (h >= p.H) break;                                        // (warp-uniform)
      const float sl = p.slope != nullptr ? p.slope[h] * MA_LOG2E : 0.f;
      float sc[KT / 32], mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < KT / 32; ++e) {
        const int c = lane + 32 * e, j = tl * KT + c;
        float v = 0.f;
#pragma unroll
        for (int s = 0; s < KSP; ++s) v += part[(static_cast<size_t>(s) * HP16 * 16 + h) * (KT + 4) + c];
        sc[e] = (j >= lo && j <= pi) ? __fmaf_rn(v, MA_LOG2E, -sl * static_cast<float>(pi - j)) : -INFINITY;
        mx = fmaxf(mx, sc[e]);
      }
#pragma unroll
      for (int d = 16; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float nm = fmaxf(m_[k], mx), mr = nm == -INFINITY ? 0.f : nm;
      const float alpha = ex2(m_[k] - mr);                        // (first tile: exp2(-inf) = 0)
      m_[k] = nm;
      float sum = 0.f;
      bf16* pr = ps + static_cast<size_t>(h / hp * per8 + h % hp) * (KT + 8);
#pragma unroll
      for (int e = 0; e < KT / 32; ++e) {
        const float w = ex2(sc[e] - mr);
        sum += w;
        pr[lane + 32 * e] = __float2bfloat16_rn(w);
      }
#pragma unroll
      for (int d = 16; d > 0; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
      l_[k] = l_[k] * alpha + sum;
      if (lane == 0) red[h] = alpha;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < MU; ++k) {
      const int u = warp + MD_WARPS * k;
      if (u >= units) break;
      const int mv = u % mtv, gn = u / mtv, g = gn / ntg, nt = gn % ntg;
      const int ha = g * hp + nt * 8 + 2 * tig, left = hp - nt * 8 - 2 * tig;            // heads of this thread's two columns
      const float a0 = left > 0 ? red[ha] : 1.f, a1 = left > 1 ? red[ha + 1] : 1.f;
      o[k][0] *= a0;
      o[k][1] *= a1;
      o[k][2] *= a0;
      o[k][3] *= a1;
      const uint32_t va = kt_a + (((lane & 7) + (lane >> 4) * 8) * rs + g * p.V + mv * 16 + ((lane >> 3) & 1) * 8) * 2;
      const uint32_t pb = ps_a + ((g * per8 + nt * 8 + gid) * (KT + 8) + 2 * tig) * 2;
#pragma unroll
      for (int c = 0; c < KT / 16; ++c) {
        uint32_t a[4], b0, b1;
        md_ldsm_t(a, va + c * 16 * rs * 2);
        asm volatile("ld.shared.b32 %0, [%1];" : "=r"(b0) : "r"(pb + c * 32));
        asm volatile("ld.shared.b32 %0, [%1];" : "=r"(b1) : "r"(pb + c * 32 + 16));
        md_mma(o[k], a, b0, b1);
      }
    }
    __syncthreads();                                              // the other buffer and P may be written again
  }
  md_wait<0>();
  // ---- merge: maximum and sum per head, unnormalised outputs; every CTA of the cluster combines a share of the outputs
#pragma unroll
  for (int k = 0; k < HP16 * 2; ++k) {
    const int h = warp + 8 * k;
    if (h < p.H && lane == 0) {
      red[MD_MAX_HEADS + h] = m_[k];
      red[2 * MD_MAX_HEADS + h] = l_[k];
    }
  }
#pragma unroll
  for (int k = 0; k < MU; ++k) {
    const int u = warp + MD_WARPS * k;
    if (u >= units) break;
    const int mv = u % mtv, gn = u / mtv, g = gn / ntg, nt = gn % ntg;
    const int ha = g * hp + nt * 8 + 2 * tig, left = hp - nt * 8 - 2 * tig;
    const int d0 = mv * 16 + gid, d1 = d0 + 8;
    if (left > 0 && d0 < p.V) outp[ha * p.V + d0] = o[k][0];
    if (left > 1 && d0 < p.V) outp[(ha + 1) * p.V + d0] = o[k][1];
    if (left > 0 && d1 < p.V) outp[ha * p.V + d1] = o[k][2];
    if (left > 1 && d1 < p.V) outp[(ha + 1) * p.V + d1] = o[k][3];
  }
  if (splits > 1) {
    __syncthreads();
    cluster_arrive_release();
    cluster_wait_acquire();
  } else {
    __syncthreads();
  }
  const int nhv = p.H * p.V, share = (nhv + splits - 1) / splits;
  const uint32_t red_a = smem_u32(red), out_a = smem_u32(outp);
  bf16* dst = p.out + static_cast<size_t>(t) * p.ld_out;
  for (int e = split * share + threadIdx.x; e < min(nhv, (split + 1) * share); e += MD_THREADS) {
    const int h = e / p.V;
    float M = -INFINITY, mm[8], num = 0.f, den = 0.f;
#pragma unroll
    for (int s = 0; s < 8; ++s) {
      if (s >= splits) break;
      mm[s] = splits > 1 ? md_ld_cluster(mapa_smem(red_a + (MD_MAX_HEADS + h) * 4, s)) : red[MD_MAX_HEADS + h];
      M = fmaxf(M, mm[s]);
    }
#pragma unroll
    for (int s = 0; s < 8; ++s) {
      if (s >= splits) break;
      const float w = ex2(mm[s] - M);                              // (a CTA without keys: exp2(-inf) = 0)
      den += w * (splits > 1 ? md_ld_cluster(mapa_smem(red_a + (2 * MD_MAX_HEADS + h) * 4, s)) : red[2 * MD_MAX_HEADS + h]);
      num += w * (splits > 1 ? md_ld_cluster(mapa_smem(out_a + e * 4, s)) : outp[e]);
    }
    dst[e] = __float2bfloat16_rn(num / den);
  }
  if (splits > 1) {                                               // nobody leaves while its shared memory is still read
    cluster_arrive_release();
    cluster_wait_acquire();
  }
}

template <int HP16, int KT, int MU>
int launch_dec(const bf16* q, const bf16* kc, const MixedArgs& a, int bytes, int seqs, int max_q, int splits, cudaStream_t s) {
  static int set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 64 || set[dev] < bytes) {
    cudaError_t e = cudaFuncSetAttribute(mixed_attention_dec_kernel<HP16, KT, MU>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         bytes);
    if (e != cudaSuccess) return static_cast<int>(e);
    if (dev < 64) set[dev] = bytes;
  }
  return static_cast<int>(launch_kernel(mixed_attention_dec_kernel<HP16, KT, MU>, dim3(max_q, seqs, splits), dim3(MD_THREADS),
                                        static_cast<size_t>(bytes), s, static_cast<unsigned>(splits), q, kc, a));
}

// what the decode kernel needs for these sizes: keys per tile (0 = not supported) and shared memory
int dec_shape(int H, int Gv, int GD, int V, int* bytes) {
  const int hp16 = H <= 16 ? 1 : (H <= 32 ? 2 : 4), per8 = (H / Gv + 7) / 8 * 8;
  const int units = Gv * ((V + 15) / 16) * (per8 / 8);
  if (H > MD_MAX_HEADS || units > MD_WARPS * 16) return 0;
  for (int kt = 64; kt >= 32; kt /= 2) {
    *bytes = md_layout(H, hp16, Gv, GD, V, kt).bytes;
    if (*bytes <= (kt == 64 ? 160 : 227) * 1024) return kt;
  }
  return 0;
}

// stages of the ring and whether the query tile stays resident; 0 = not supported
int tc_shape(int GD, int V, bool* qres, int* bytes) {
  const int ns = (GD + 63) / 64;
  const int nv_max = V % 64 == 0 ? V / 64 : (V + 63 - 1) / 64 + 1;          // value slabs a head may touch
  if (V > 128 || 2 * MT_BKV + nv_max * 64 > 512) return 0;
  int nst = (MT_SMEM_MAX - MT_BAR_BYTES - ns * MT_SLAB) / MT_SLAB;
  *qres = nst >= 4;
  const int stage = *qres ? MT_SLAB : 2 * MT_SLAB;
  if (!*qres) nst = (MT_SMEM_MAX - MT_BAR_BYTES) / stage;
  nst = nst < MT_MAX_STAGES ? nst : MT_MAX_STAGES;
  *bytes = (*qres ? ns * MT_SLAB : 0) + nst * stage + MT_BAR_BYTES;
  return nst;
}

}  // namespace

bool mixed_attention_supported(int H, int Gv, int GD, int V) {
  bool qres;
  int bytes;
  return H > 0 && Gv > 0 && H % Gv == 0 && GD == Gv * V && GD % 8 == 0 && V % 8 == 0 && tc_shape(GD, V, &qres, &bytes) > 0;
}

int launch_mixed_attention(const void* q, int q_rows, const void* k_cache, int n_pages, void* out, int ld_out,
                           const int* block_table, int max_pages, const int* q_start, const int* q_len, const int* kv_len,
                           int n_seqs, int max_q, int H, int Gv, int GD, int V, int window, const float* slope,
                           const float* sink, cudaStream_t s) {
  if (n_seqs <= 0 || max_q <= 0) return 0;
  if (!mixed_attention_supported(H, Gv, GD, V) || ld_out % 8 != 0 || reinterpret_cast<uintptr_t>(out) % 16 != 0) return -2;
  MixedArgs a{};
  a.out = static_cast<bf16*>(out);
  a.block_table = block_table; a.q_start = q_start; a.q_len = q_len; a.kv_len = kv_len;
  a.slope = slope; a.sink = sink;
  a.ld_out = ld_out; a.max_pages = max_pages; a.H = H; a.Gv = Gv; a.GD = GD; a.V = V; a.window = window;
  int dbytes = 0;
  const int kt = max_q <= 2 ? dec_shape(H, Gv, GD, V, &dbytes) : 0;
  if (kt > 0) {
    // CTAs per query: enough to give every SM one (clusters of up to 8), no more than the window has tiles
    const int resident = dbytes <= 110 * 1024 ? 2 * 148 : 148;
    int splits = 1;
    while (splits < 8 && n_seqs * max_q * splits * 2 <= resident && (window <= 0 || window > splits * kt)) splits *= 2;
    const bf16* qb = static_cast<const bf16*>(q);
    const bf16* kb = static_cast<const bf16*>(k_cache);
    const int hp16 = H <= 16 ? 1 : (H <= 32 ? 2 : 4);
    const int units = Gv * ((V + 15) / 16) * ((H / Gv + 7) / 8);
    const bool wide = units > MD_WARPS * 8;
#define B2B_MD(HP, KT_)                                                                                                 \
  if (hp16 == HP && kt == KT_)                                                                                          \
    return wide ? launch_dec<HP, KT_, 16>(qb, kb, a, dbytes, n_seqs, max_q, splits, s)                                  \
                : launch_dec<HP, KT_, 8>(qb, kb, a, dbytes, n_seqs, max_q, splits, s);
    B2B_MD(1, 64) B2B_MD(1, 32) B2B_MD(2, 64) B2B_MD(2, 32) B2B_MD(4, 64) B2B_MD(4, 32)
#undef B2B_MD
  }
  bool qres;
  int bytes;
  a.nst = tc_shape(GD, V, &qres, &bytes);
  a.ns = (GD + 63) / 64;
  CUtensorMap tq, tk;
  int r = make_tmap_shared(&tq, q, static_cast<uint64_t>(q_rows), static_cast<uint64_t>(H) * GD, static_cast<uint64_t>(H) * GD,
                           128, 2);
  if (r) return r;
  if ((r = make_tmap_shared(&tk, k_cache, static_cast<uint64_t>(n_pages) * MA_PAGE, static_cast<uint64_t>(GD),
                            static_cast<uint64_t>(GD), MA_PAGE, 2)))
    return r;
  static bool set[2][64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 64 || !set[qres][dev]) {
    cudaError_t e = qres ? cudaFuncSetAttribute(mixed_attention_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, MT_SMEM_MAX)
                         : cudaFuncSetAttribute(mixed_attention_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, MT_SMEM_MAX);
    if (e != cudaSuccess) return static_cast<int>(e);
    if (dev < 64) set[qres][dev] = true;
  }
  const dim3 grid((max_q + 127) / 128, H, n_seqs);
  return static_cast<int>(qres ? launch_kernel(mixed_attention_tc_kernel<true>, grid, dim3(MT_THREADS), static_cast<size_t>(bytes), s, 1u,
                                               tq, tk, a)
                               : launch_kernel(mixed_attention_tc_kernel<false>, grid, dim3(MT_THREADS), static_cast<size_t>(bytes), s, 1u,
                                               tq, tk, a));
}

unsigned mixed_attention_gave_up() {
  unsigned n = 0;
  return cudaMemcpyFromSymbol(&n, g_mixed_gave_up, sizeof(n)) == cudaSuccess ? n : ~0u;
}

int set_wait_policy_mixed(uint32_t* abort_word, unsigned long long limit_ns) {
  cudaError_t e = cudaMemcpyToSymbol(g_abort_word, &abort_word, sizeof(abort_word));
  if (e == cudaSuccess) e = cudaMemcpyToSymbol(g_wait_limit_ns, &limit_ns, sizeof(limit_ns));
  return static_cast<int>(e);
}

}  // namespace b2b
