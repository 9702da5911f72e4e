// Differential softmax attention over the paged KV cache, bf16 serving mode (float32 mode and other sizes run the exact
// softmax_attention kernel of seqmix.cu and diff_combine).  A head has two query / key maps of D channels over the SAME values:
//     out[i, h, :] = d / rms(d) * gain,  d = softmax(q_1 . k_1) v - lambda softmax(q_2 . k_2) v
// over the keys j <= i, and j > i - window when window > 0.
//
// One CTA = the query heads that share a key/value head (hg of them, stacked into the 128 rows of a tile: row = (query, head of the
// group)) for up to 128 / hg consecutive queries.  Both maps of the group live in one CTA: scores S_1, S_2 and outputs O_1, O_2
// fill the 512 columns of tensor memory, a value tile is fetched once for both, and while the softmax threads of one map work,
// the tensor cores compute the other map's products.  Key and value tiles of 128 rows come by TMA in slabs of 64 channels
// through a ring of 16 KB stages.  Warp roles: 0 TMA producer, 1 MMA issuer, 2..5 softmax of map 1, 6..9 of map 2 (a thread owns one
// row).  P overwrites its scores as the TMEM operand of the second product.  The combination, the norm over the head and the
// bf16 rows are the epilogue.
// Decode steps (one or two tokens per sequence): the same kernel with few live rows; when sequences x key/value heads do not fill
// the machine, a cluster of CTAs shares the keys of a tile and merges the partial results through distributed shared memory.
// Scores, masks, maxima, sums and the combination are fp32; P is rounded to bf16 as the operand of the second product.  Every wait
// is bounded: one that runs out raises the abort word of the engine, and the CTA drains its copies, frees its tensor memory and leaves.
// This translation unit is compiled WITHOUT --use_fast_math; the exponentials are the hardware exp2 (2^-22 relative).
#include "kernels.h"

#include <cuda.h>

#include <map>
#include <mutex>
#include <tuple>
#include <type_traits>

#include "common.cuh"
#include "launch.cuh"
#include "tmem.cuh"

namespace b2b {
namespace {

typedef __nv_bfloat16 bf16;
constexpr int DA_PAGE = 64, DA_BKV = 128, DA_THREADS = 320;
constexpr int DA_SLAB = 128 * 128;                  // 128 rows x 64 channels, 128-byte swizzle
constexpr int DA_MAX_STAGES = 13;
constexpr int DA_SMEM_MAX = 227 * 1024;
constexpr int DA_AUX = 512 + 2 * 2 * 128 * 4;       // barriers | per map and row: reference maximum, sum (or partial square sums)
constexpr int DA_SPLIT_ROWS = 32;                   // rows a cluster may merge

struct DiffArgs {
  bf16* out;
  const int* block_table;
  const int* q_start;
  const int* q_len;
  const int* kv_len;
  float lambda, gain, eps;
  int ld_out, max_pages, G, hg, V, window;
  int ns, nv, nst, nq, splits;      // slabs of a key map / of a value row, ring stages, queries per CTA, CTAs per cluster
};

__device__ unsigned int g_diff_gave_up = 0;         // CTAs whose waits ran out since the module was loaded

__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* m, uint64_t* bar, int c0, int c1, int c2) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2)
      : "memory");
}
__device__ __forceinline__ float ld_cluster_f32(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}

// grid (query tiles, key/value heads, sequences x splits), cluster (1, 1, splits)
__global__ void __launch_bounds__(DA_THREADS, 1)
    diff_attention_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                          const __grid_constant__ CUtensorMap tm_v, const DiffArgs p) {
  constexpr uint32_t S_COL = 0, O_COL = 2 * DA_BKV, TCOLS = 512;       // columns of map m: S_COL + 128 m, O_COL + 128 m
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* q_s = smem;                                                 // [2 maps][ns] slabs
  uint8_t* ring = smem + 2 * p.ns * DA_SLAB;                           // [nst] slabs
  uint64_t* bars = reinterpret_cast<uint64_t*>(ring + p.nst * DA_SLAB);
  uint64_t* full = bars;
  uint64_t* empty = bars + DA_MAX_STAGES;
  uint64_t* s_full = bars + 2 * DA_MAX_STAGES;                         // [2 maps]
  uint64_t* p_ready = s_full + 2;
  uint64_t* pv_done = s_full + 4;
  uint64_t* q_full = s_full + 6;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(s_full + 7);
  volatile uint32_t* abort = tmem_slot + 1;
  volatile uint32_t* issued = tmem_slot + 2;                           // slabs the producer has asked for
  float* row_m = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(bars) + 512);      // [2 maps][128] reference maximum / square sums
  float* row_l = row_m + 2 * 128;                                      // [2 maps][128] sums

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < p.nst; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    for (int m = 0; m < 2; ++m) {
      mbar_init(&s_full[m], 1);
      mbar_init(&p_ready[m], 4);
      mbar_init(&pv_done[m], 1);
    }
    mbar_init(q_full, 1);
    *abort = 0u;
    *issued = 0u;
    fence_barrier_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 1) tmem_alloc<TCOLS>(tmem_slot);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  pdl_launch_dependents();                                             // (every CTA of the grid owns its tensor memory by then)
  pdl_wait();

  const int seq = blockIdx.z / p.splits, split = blockIdx.z % p.splits, g = blockIdx.y;
  const int qlen = p.q_len[seq], kvlen = p.kv_len[seq];
  const int q0 = blockIdx.x * p.nq;
  const bool active = q0 < qlen;                                       // uniform over the cluster
  const int nqv = min(p.nq, qlen - q0), n_rows = nqv * p.hg;
  const int qtok0 = p.q_start[seq] + q0;
  const int pos0 = kvlen - qlen + q0;                                  // position of the tile's first query
  const int kv_hi = pos0 + nqv;
  const int kv_lo = p.window > 0 ? max(0, pos0 - p.window + 1) : 0;
  int t_lo = kv_lo / DA_BKV;
  int nt = active ? (kv_hi + DA_BKV - 1) / DA_BKV - t_lo : 0;
  if (p.splits > 1) {                                                  // this CTA's share of the key tiles (possibly none)
    const int each = (nt + p.splits - 1) / p.splits, tb = min(nt, split * each), te = min(nt, tb + each);
    t_lo += tb;
    nt = te - tb;
  }
  auto all = [](bool b) { return __all_sync(0xffffffffu, b) != 0; };

  if (nt == 0) {
    if (warp >= 2) {                                                   // (only the merge of a cluster reads these)
      const int m = (warp - 2) >> 2, i = (warp & 3) * 32 + lane;
      row_m[m * 128 + i] = -INFINITY;
      row_l[m * 128 + i] = 0.f;
    }
  } else if (warp == 0) {
    if (elect_one()) {
      mbar_arrive_expect_tx(q_full, 2 * p.ns * p.nq * p.hg * 128);
      for (int m = 0; m < 2; ++m)
        for (int c = 0; c < p.ns; ++c)
          tma_load_3d(q_s + (m * p.ns + c) * DA_SLAB, &tm_q, q_full, c * 64, (g * 2 + m) * p.hg, qtok0);
      const int* bt = p.block_table + static_cast<size_t>(seq) * p.max_pages;
      int st = 0;
      uint32_t ph = 0, cnt = 0;
      auto slabs = [&](const CUtensorMap* tm, int n, int row, int cn) {
        const int pg = 2 * (t_lo + n);
        const int page0 = bt[pg];
        const int page1 = (pg + 1 < p.max_pages && (pg + 1) * DA_PAGE < kv_hi) ? bt[pg + 1] : page0;   // past the newest key: any rows
        for (int c = 0; c < cn; ++c) {
          if (!ma_wait(&empty[st], ph ^ 1u, abort)) return false;
          uint8_t* dst = ring + st * DA_SLAB;
          mbar_arrive_expect_tx(&full[st], DA_SLAB);
          tma_load_3d(dst, tm, &full[st], c * 64, row, page0 * DA_PAGE);
          tma_load_3d(dst + DA_SLAB / 2, tm, &full[st], c * 64, row, page1 * DA_PAGE);
          *issued = ++cnt;
          if (++st == p.nst) {
            st = 0;
            ph ^= 1u;
          }
        }
        return true;
      };
      bool ok = slabs(&tm_k, 0, 2 * g, p.ns) && slabs(&tm_k, 0, 2 * g + 1, p.ns);
      for (int n = 0; n < nt && ok; ++n) {                             // the order in which the MMA warp consumes
        ok = slabs(&tm_v, n, g, p.nv);
        if (n + 1 < nt) ok = ok && slabs(&tm_k, n + 1, 2 * g, p.ns) && slabs(&tm_k, n + 1, 2 * g + 1, p.ns);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    constexpr uint32_t idesc_s = make_idesc_bf16(128, DA_BKV);
    constexpr uint32_t idesc_o = make_idesc_bf16(128, 64) | (1u << 16);      // B operand (values) is MN-major
    int st = 0;
    uint32_t ph = 0;
    auto next = [&] {
      if (++st == p.nst) {
        st = 0;
        ph ^= 1u;
      }
    };
    auto qk = [&](int m) {                                             // scores of map m against the ring's next slabs
      for (int i = 0; i < p.ns; ++i) {
        if (!all(ma_wait(&full[st], ph, abort))) return false;
        tc_fence_after();
        if (elect_one()) {
          const uint32_t ks = smem_u32(ring + st * DA_SLAB), qs = smem_u32(q_s + (m * p.ns + i) * DA_SLAB);
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            umma_bf16(tmem + S_COL + m * DA_BKV, make_sw128_kmajor_desc(qs) + static_cast<uint64_t>(kk * 2),
                      make_sw128_kmajor_desc(ks) + static_cast<uint64_t>(kk * 2), idesc_s, (i > 0 || kk > 0) ? 1u : 0u);
          umma_commit(&empty[st]);
          if (i == p.ns - 1) umma_commit(&s_full[m]);
        }
        __syncwarp();
        next();
      }
      return true;
    };
    auto pv = [&](int m, int n, int v_st) {                            // outputs of map m; the second map releases the value slabs
      for (int j = 0; j < p.nv; ++j) {
        const int s = v_st + j < p.nst ? v_st + j : v_st + j - p.nst;
        if (elect_one()) {
          const uint32_t vb = smem_u32(ring + s * DA_SLAB);
#pragma unroll
          for (int kk = 0; kk < DA_BKV / 16; ++kk)
            ma_mma_ts(tmem + O_COL + m * 128 + j * 64, tmem + S_COL + m * DA_BKV + kk * 8, ma_value_desc(vb + kk * (16 * 128)), idesc_o,
                      (n > 0 || kk > 0) ? 1u : 0u);
          if (m == 1) umma_commit(&empty[s]);
          if (j == p.nv - 1) umma_commit(&pv_done[m]);
        }
        __syncwarp();
      }
    };
    bool ok = all(ma_wait(q_full, 0, abort));
    ok = ok && qk(0) && qk(1);
    for (int n = 0; n < nt && ok; ++n) {
      const int v_st = st;
      for (int j = 0; j < p.nv && ok; ++j) {
        ok = all(ma_wait(&full[st], ph, abort));
        next();
      }
      for (int m = 0; m < 2 && ok; ++m) {
        if (!(ok = all(ma_wait(&p_ready[m], static_cast<uint32_t>(n & 1), abort)))) break;
        tc_fence_after();
        pv(m, n, v_st);
        if (n + 1 < nt) ok = qk(m);                                    // runs under the other map's softmax
      }
    }
  } else {
    const int quarter = warp & 3, m = (warp - 2) >> 2;
    const int i = quarter * 32 + lane;                                 // row of the tile
    const bool row_valid = i < n_rows;
    const int qi = i / p.hg, qpos = pos0 + qi;
    const int lo = p.window > 0 ? qpos - p.window + 1 : 0;
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(quarter * 32) << 16);
    const uint32_t s_addr = lane_addr + S_COL + m * DA_BKV, o_addr = lane_addr + O_COL + m * 128;
    float m_ref = -INFINITY, l = 0.f;

    auto tile = [&](int n, auto masked) {
      const int kb = (t_lo + n) * DA_BKV;
      if (!all(ma_wait(&s_full[m], static_cast<uint32_t>(n & 1), abort))) return false;
      if (quarter * 32 >= n_rows) {                                    // (warp-uniform; decode steps: what its rows hold is never read)
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_ready[m]);
        return true;
      }
      tc_fence_after();
      uint32_t r[DA_BKV];
#pragma unroll
      for (int c = 0; c < DA_BKV; c += 32) ma_ld32(s_addr + c, r + c);
#pragma unroll
      for (int c = 0; c < DA_BKV; c += 32) ma_ld_fence(r + c);
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int e = 0; e < DA_BKV; ++e) {
        if constexpr (decltype(masked)::value) {
          const int j = kb + e;
          if (!(row_valid && j <= qpos && j >= lo)) r[e] = __float_as_uint(-INFINITY);
        }
        mx4[e & 3] = fmaxf(mx4[e & 3], __uint_as_float(r[e]));
      }
      const float mrow = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      // lazy rescaling: the reference stays while the new maximum is within 2^8 of it
      float alpha = 1.f;
      if (mrow > m_ref + 8.f || (m_ref == -INFINITY && mrow > -INFINITY)) {
        alpha = (m_ref == -INFINITY) ? 0.f : ex2(m_ref - mrow);
        m_ref = mrow;
      }
      const float mr = (m_ref == -INFINITY) ? 0.f : m_ref;             // nothing visible so far: exp2(-inf) = 0
      float ls[2] = {0.f, 0.f};
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        uint32_t pk[32];
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          const float p0 = ex2(__uint_as_float(r[64 * hf + 2 * j]) - mr);
          const float p1 = ex2(__uint_as_float(r[64 * hf + 2 * j + 1]) - mr);
          ls[j & 1] += p0 + p1;
          pk[j] = pack2(p0, p1);
        }
        ma_st32(s_addr + hf * 32, pk);                                 // over the scores of this tile, which are in registers
      }
      if (n > 0) {
        if (!all(ma_wait(&pv_done[m], static_cast<uint32_t>((n - 1) & 1), abort))) return false;
        tc_fence_after();
        if (__any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll 1
          for (int c = 0; c < p.nv * 64; c += 32) {
            uint32_t o[32];
            ma_ld32(o_addr + c, o);
            ma_ld_fence(o);
#pragma unroll
            for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * alpha);
            ma_st32(o_addr + c, o);
          }
        }
      }
      ma_st_wait();
      l = l * alpha + (ls[0] + ls[1]);
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_ready[m]);
      return true;
    };

    bool ok = true;
    for (int n = 0; n < nt && ok; ++n) {
      const int kb = (t_lo + n) * DA_BKV;
      const bool every = n_rows == 128 && kb + DA_BKV - 1 <= pos0 && (p.window <= 0 || kb > pos0 + nqv - 1 - p.window);
      ok = every ? tile(n, std::false_type{}) : tile(n, std::true_type{});
    }
    row_l[m * 128 + i] = l;
    if (p.splits > 1) {
      // partial result of this CTA: unnormalised rows in place of the ring (every slab has been consumed)
      row_m[m * 128 + i] = m_ref;
      if (ok) ok = all(ma_wait(&pv_done[0], static_cast<uint32_t>((nt - 1) & 1), abort)) &&
                   all(ma_wait(&pv_done[1], static_cast<uint32_t>((nt - 1) & 1), abort));
      asm volatile("bar.sync 1, 256;" ::: "memory");
      if (ok && quarter * 32 < n_rows) {
        tc_fence_after();
        float* part = reinterpret_cast<float*>(ring) + static_cast<size_t>(m * DA_SPLIT_ROWS + i) * p.V;
#pragma unroll 1
        for (int c = 0; c < p.V; c += 32) {
          uint32_t o[32];
          ma_ld32(o_addr + c, o);
          ma_ld_fence(o);
          if (!row_valid) continue;
#pragma unroll
          for (int e = 0; e < 32; e += 4)
            if (c + e < p.V)
              *reinterpret_cast<float4*>(part + c + e) = make_float4(__uint_as_float(o[e]), __uint_as_float(o[e + 1]),
                                                                     __uint_as_float(o[e + 2]), __uint_as_float(o[e + 3]));
        }
      }
    } else {
      if (ok) ok = all(ma_wait(&pv_done[0], static_cast<uint32_t>((nt - 1) & 1), abort)) &&
                   all(ma_wait(&pv_done[1], static_cast<uint32_t>((nt - 1) & 1), abort));
      asm volatile("bar.sync 1, 256;" ::: "memory");                   // (every softmax warp takes part, aborted or not)
      tc_fence_after();
      const float l1 = row_l[i], l2 = row_l[128 + i];
      const float c1 = l1 > 0.f ? 1.f / l1 : 0.f, c2 = l2 > 0.f ? p.lambda / l2 : 0.f;
      const uint32_t oa = lane_addr + O_COL;
      // the two threads of a row (one per map) share its channels in chunks of 32: sum of squares, then the normed rows
      float ss = 0.f;
      if (ok) {
#pragma unroll 1
        for (int c = 32 * m; c < p.V; c += 64) {
          uint32_t a[32], b[32];
          ma_ld32(oa + c, a);
          ma_ld32(oa + 128 + c, b);
          ma_ld_fence(a);
          ma_ld_fence(b);
#pragma unroll
          for (int e = 0; e < 32; ++e) {                               // (channels behind V are zero)
            const float d = __uint_as_float(a[e]) * c1 - __uint_as_float(b[e]) * c2;
            ss += d * d;
          }
        }
      }
      row_m[m * 128 + i] = ss;
      asm volatile("bar.sync 1, 256;" ::: "memory");
      if (ok) {
        const float k = p.gain / sqrtf((row_m[i] + row_m[128 + i]) / static_cast<float>(p.V) + p.eps);
        bf16* dst = p.out + static_cast<size_t>(qtok0 + qi) * p.ld_out + (g * p.hg + i - qi * p.hg) * p.V;
#pragma unroll 1
        for (int c = 32 * m; c < p.V; c += 64) {
          uint32_t a[32], b[32];
          ma_ld32(oa + c, a);
          ma_ld32(oa + 128 + c, b);
          ma_ld_fence(a);
          ma_ld_fence(b);
          if (!row_valid) continue;
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            if (c + 8 * j >= p.V) break;
            uint32_t w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int x = 8 * j + 2 * e;
              w[e] = pack2((__uint_as_float(a[x]) * c1 - __uint_as_float(b[x]) * c2) * k,
                           (__uint_as_float(a[x + 1]) * c1 - __uint_as_float(b[x + 1]) * c2) * k);
            }
            *reinterpret_cast<uint4*>(dst + c + 8 * j) = make_uint4(w[0], w[1], w[2], w[3]);
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (nt > 0 && *abort != 0u) {
    // a wait ran out: report it, let the copies that are still in flight land (again bounded), leave
    if (threadIdx.x == 0) {
      if (g_abort_word != nullptr) *g_abort_word = 1u;
      atomicAdd(&g_diff_gave_up, 1u);
      const uint32_t n = *issued;
      for (int s = 0; s < p.nst; ++s) {
        if (n <= static_cast<uint32_t>(s)) break;
        const uint32_t uses = (n - s - 1) / p.nst;                     // the stage's last phase
        for (uint32_t k = 0; k < (1u << 20) && !mbar_try_wait(&full[s], uses & 1u); ++k) {}
      }
      for (uint32_t k = 0; k < (1u << 20) && !mbar_try_wait(q_full, 0); ++k) {}
    }
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc<TCOLS>(tmem);
  }
  if (p.splits > 1 && active) {                                        // (uniform over the cluster)
    cluster_arrive_release();
    cluster_wait_acquire();
    // rows split, split + splits, ...: one warp each; partial rows are weighted by exp2 of their maxima
    const uint32_t rm = smem_u32(row_m), rl = smem_u32(row_l), pa = smem_u32(ring);
    for (int i = split + p.splits * warp; i < n_rows; i += p.splits * (DA_THREADS / 32)) {
      float w[2][8], inv[2];
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        float mx = -INFINITY, den = 0.f;
#pragma unroll
        for (int s = 0; s < 8; ++s) {
          w[m][s] = s < p.splits ? ld_cluster_f32(mapa_smem(rm + (m * 128 + i) * 4, s)) : -INFINITY;
          mx = fmaxf(mx, w[m][s]);
        }
#pragma unroll
        for (int s = 0; s < 8; ++s) {                                  // (a CTA without keys: exp2(-inf) = 0)
          w[m][s] = ex2(w[m][s] - mx);
          if (s < p.splits && w[m][s] > 0.f) den += w[m][s] * ld_cluster_f32(mapa_smem(rl + (m * 128 + i) * 4, s));
        }
        inv[m] = 1.f / den;
      }
      inv[1] *= p.lambda;
      float d[4], ss = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int c = lane + 32 * k;
        d[k] = 0.f;
        if (c >= p.V) continue;
        float a = 0.f, b = 0.f;
#pragma unroll
        for (int s = 0; s < 8; ++s) {
          if (s >= p.splits) break;
          if (w[0][s] > 0.f) a += w[0][s] * ld_cluster_f32(mapa_smem(pa + (i * p.V + c) * 4, s));
          if (w[1][s] > 0.f) b += w[1][s] * ld_cluster_f32(mapa_smem(pa + ((DA_SPLIT_ROWS + i) * p.V + c) * 4, s));
        }
        d[k] = a * inv[0] - b * inv[1];
        ss += d[k] * d[k];
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float k = p.gain / sqrtf(ss / static_cast<float>(p.V) + p.eps);
      const int qi = i / p.hg;
      bf16* dst = p.out + static_cast<size_t>(qtok0 + qi) * p.ld_out + (g * p.hg + i - qi * p.hg) * p.V;
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (lane + 32 * j < p.V) dst[lane + 32 * j] = __float2bfloat16_rn(d[j] * k);
    }
    cluster_arrive_release();                                          // nobody leaves while its shared memory is still read
    cluster_wait_acquire();
  }
}

using PFN_encodeTiled = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                     const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                     CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// bf16 [rows][heads][chans], box 64 channels x box_heads x box_rows, 128-byte swizzle, zeros outside
int make_tmap3(CUtensorMap* m, const void* ptr, uint64_t rows, uint64_t heads, uint64_t chans, uint32_t box_heads, uint32_t box_rows) {
  using Key = std::tuple<const void*, uint64_t, uint64_t, uint64_t, uint32_t, uint32_t>;
  static std::map<Key, CUtensorMap> cache;
  static std::mutex mu;
  static PFN_encodeTiled enc = nullptr;
  std::lock_guard<std::mutex> lock(mu);
  const Key key{ptr, rows, heads, chans, box_heads, box_rows};
  const auto it = cache.find(key);
  if (it != cache.end()) {
    *m = it->second;
    return 0;
  }
  if (enc == nullptr) {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult res;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &res) != cudaSuccess || res != cudaDriverEntryPointSuccess)
      return -1;
    enc = reinterpret_cast<PFN_encodeTiled>(fn);
  }
  const cuuint64_t dims[3] = {chans, heads, rows}, strides[2] = {chans * 2, chans * heads * 2};
  const cuuint32_t box[3] = {64, box_heads, box_rows}, est[3] = {1, 1, 1};
  const CUresult r = enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, est,
                         CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                         CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return static_cast<int>(r);
  if (cache.size() > 65536) cache.clear();
  cache[key] = *m;
  return 0;
}

// stages of the ring, 0 = sizes the kernel does not have
int ring_stages(int D, int V) {
  const int ns = (D + 63) / 64, nv = (V + 63) / 64;
  int n = (DA_SMEM_MAX - DA_AUX - 2 * ns * DA_SLAB) / DA_SLAB;
  if (n > DA_MAX_STAGES) n = DA_MAX_STAGES;
  return n >= ns + nv ? n : 0;
}

}  // namespace

bool diff_attention_supported(int H, int G, int D, int V) {
  return H > 0 && G > 0 && H % G == 0 && H / G <= 128 && D > 0 && V > 0 && D % 8 == 0 && V % 8 == 0 && D <= 128 && V <= 128 &&
         ring_stages(D, V) > 0;
}

int launch_diff_attention(const void* q, int q_rows, const void* k_cache, const void* v_cache, int n_pages, void* out, int ld_out,
                          const int* block_table, int max_pages, const int* q_start, const int* q_len, const int* kv_len, int n_seqs,
                          int max_q, int H, int G, int D, int V, int window, float lambda, float gain, float eps, cudaStream_t s) {
  if (n_seqs <= 0 || max_q <= 0) return 0;
  auto al16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  if (!diff_attention_supported(H, G, D, V) || ld_out % 8 != 0 || !al16(out) || !al16(q) || !al16(k_cache) || !al16(v_cache)) return -2;
  DiffArgs a{};
  a.out = static_cast<bf16*>(out);
  a.block_table = block_table; a.q_start = q_start; a.q_len = q_len; a.kv_len = kv_len;
  a.lambda = lambda; a.gain = gain; a.eps = eps;
  a.ld_out = ld_out; a.max_pages = max_pages; a.G = G; a.hg = H / G; a.V = V; a.window = window;
  a.ns = (D + 63) / 64; a.nv = (V + 63) / 64; a.nst = ring_stages(D, V);
  a.nq = 128 / a.hg < max_q ? 128 / a.hg : max_q;
  a.splits = 1;
  const int tiles = (max_q + a.nq - 1) / a.nq;
  if (a.nq * a.hg <= DA_SPLIT_ROWS && max_q <= 2) {
    // decode steps: enough CTAs to give every SM one (clusters of up to 8), no more than there can be key tiles
    const int keys = window > 0 && window < max_pages * DA_PAGE ? window : max_pages * DA_PAGE;
    while (a.splits < 8 && static_cast<long long>(tiles) * G * n_seqs * a.splits * 2 <= 148 && keys > a.splits * DA_BKV) a.splits *= 2;
  }
  CUtensorMap tq, tk, tv;
  int r = make_tmap3(&tq, q, static_cast<uint64_t>(q_rows), 2 * static_cast<uint64_t>(H), static_cast<uint64_t>(D),
                     static_cast<uint32_t>(a.hg), static_cast<uint32_t>(a.nq));
  if (r) return r;
  const uint64_t rows = static_cast<uint64_t>(n_pages) * DA_PAGE;
  if ((r = make_tmap3(&tk, k_cache, rows, 2 * static_cast<uint64_t>(G), static_cast<uint64_t>(D), 1, DA_PAGE))) return r;
  if ((r = make_tmap3(&tv, v_cache, rows, static_cast<uint64_t>(G), static_cast<uint64_t>(V), 1, DA_PAGE))) return r;
  static bool set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 64 || !set[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(diff_attention_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, DA_SMEM_MAX);
    if (e != cudaSuccess) return static_cast<int>(e);
    if (dev < 64) set[dev] = true;
  }
  const size_t bytes = static_cast<size_t>(2 * a.ns + a.nst) * DA_SLAB + DA_AUX;
  return static_cast<int>(launch_kernel(diff_attention_kernel, dim3(tiles, G, n_seqs * a.splits), dim3(DA_THREADS), bytes, s,
                                        static_cast<unsigned>(a.splits), tq, tk, tv, a));
}

unsigned diff_attention_gave_up() {
  unsigned n = 0;
  return cudaMemcpyFromSymbol(&n, g_diff_gave_up, sizeof(n)) == cudaSuccess ? n : ~0u;
}

int set_wait_policy_diff(uint32_t* abort_word, unsigned long long limit_ns) {
  cudaError_t e = cudaMemcpyToSymbol(g_abort_word, &abort_word, sizeof(abort_word));
  if (e == cudaSuccess) e = cudaMemcpyToSymbol(g_wait_limit_ns, &limit_ns, sizeof(limit_ns));
  return static_cast<int>(e);
}

}  // namespace b2b
