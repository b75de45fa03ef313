// Absorbed latent decode on the 5th-generation tensor cores (tcgen05 + TMEM + TMA), for pools of 16-token blocks.
//
// With 16 or 32 heads on the N side of the instruction no tile row is padding: a CTA owns (sequence, tile of N heads, KV
// split) and walks the split in tiles of 64 tokens,
//   scores  S^T [64 tokens, N]   = rows [64, W] x queries [N, W]^T     (M = 64; both K-major, as TMA lands them)
//   values  O^T [128 columns, N] += rows [64 tokens, 128 columns]^T x weights [N, 64 tokens]^T, per 128 latent columns
//                                   (the SAME shared tile, read MN-major)
//
//   warp 0 and the last two: TMA producers, taking slots in turn: the queries once; per tile ceil(W / 128) slots of [64 tokens][128 columns] (two 64-column
//              128-byte-swizzled sub-tiles, four pool blocks each) through a ring that holds at least two tiles where it
//              can; a slot of latent columns is free again when its value MMA has run, one of the rotated part already
//              after the scores
//   warp 1     MMA issuer; the scores of tile j + 1 run under the softmax of tile j (S and the weights are double-buffered)
//   warps 2..  softmax, four warps per 16 heads, one token per thread: running maxima per head by integer warp reductions
//              on order-preserving bits and one exchange through shared memory, lazy rescaling of O (only when a maximum
//              grows by more than 2^8), weights as two bf16 terms (rounded weight and remainder) that sit side by side on
//              the N side, so the value rows are read once for both; the epilogue, one latent column per thread
//
// Every wait is bounded and reports through the status word. Barriers that tiles use in turn come in pairs, so that none
// can be two phases past the one a thread waits for. Splits leave fp32 partial results for latent_merge_kernel.
#include "api.h"
#include "latent.cuh"

namespace mx {

bool make_tensor_map_bf16(CUtensorMap* out, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows,
                          uint32_t box_cols);
bool make_tensor_map_bf16_3d(CUtensorMap* out, const void* ptr, uint64_t rows, uint64_t groups, uint64_t cols, uint64_t ld,
                             uint64_t group_ld, uint32_t box_rows, uint32_t box_cols);

constexpr int kLtKeys = 64, kLtBlock = 16;
constexpr int kLtHeads = 16;                         // heads per softmax thread
constexpr int kLtProducers = 3;                      // one warp's issue rate does not keep up with boxes of one pool block
__host__ __device__ constexpr int lt_threads(int N) { return 32 * (1 + kLtProducers) + 128 * (N / kLtHeads); }
constexpr int kLtSub = kLtKeys * 128;                // one [64 tokens][64 columns] sub-tile
constexpr int kLtSlot = 2 * kLtSub;
constexpr int kLtMaxSlots = 20;
constexpr float kLtRescale = 8.0f;                   // log2 units

enum : int { kErrLatentProducer = 411, kErrLatentMma = 412, kErrLatentSoftmax = 413 };

struct LatentTcParams {
  LatentDecodeParams d;
  int* status;
  int slots;                                         // ring depth
};

__host__ inline int lt_fixed_smem(int W, int N) {    // queries, weights, control words, alignment
  return (W + 63) / 64 * N * 128 + 4 * N * 128 + 2560 + 1024;
}

// Order-preserving map between floats and signed integers (its own inverse).
__device__ __forceinline__ int float_order(int bits) { return bits ^ ((bits >> 31) & 0x7FFFFFFF); }

template <int N>
__global__ void __launch_bounds__(lt_threads(N), 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_pool, const LatentTcParams t) {
  constexpr uint32_t TMEM_COLS = N <= 16 ? 256 : 512;   // S: two buffers of 4 N columns; O: up to four blocks of 2 N (N per term)
  constexpr int O_COL = 8 * N, Q_SUB = N * 128, P_SUB = 2 * N * 128, GROUPS = N / kLtHeads, HT = kLtHeads;
  const LatentDecodeParams& p = t.d;
  extern __shared__ uint8_t lt_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lt_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int subs = (p.W + 63) / 64, np = (p.W + 127) / 128, nm = (p.C + 127) / 128;
  uint8_t* k_sm = smem;                              // slots x kLtSlot
  uint8_t* q_sm = k_sm + t.slots * kLtSlot;          // subs x Q_SUB
  uint8_t* p_sm = q_sm + subs * Q_SUB;               // [2 buffers][2 terms][N rows of 128 bytes]
  uint64_t* bars = reinterpret_cast<uint64_t*>(p_sm + 2 * P_SUB);
  uint64_t *full = bars, *empty = full + kLtMaxSlots, *q_full = empty + kLtMaxSlots, *s_full = q_full + 1, *p_full = s_full + 2,
           *pv_done = p_full + 2, *swap_bar = pv_done + 2;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(swap_bar + GROUPS);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x % p.num_splits, bt = blockIdx.x / p.num_splits;
  const int ht = bt % p.head_tiles, b = bt / p.head_tiles, h0 = ht * N;
  const int len = p.context_lens[b];
  const LatentSpan span = latent_span(p, len, split, kLtKeys);
  const int t0 = span.t0, n_tiles = max(0, span.t1 - t0);

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_pool);
    for (int i = 0; i < t.slots; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(q_full, 1);
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    mbar_init(&p_full[0], 4 * GROUPS);
    mbar_init(&p_full[1], 4 * GROUPS);
    mbar_init(&pv_done[0], 1);
    mbar_init(&pv_done[1], 1);
    for (int i = 0; i < GROUPS; ++i) mbar_init(&swap_bar[i], 4);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_ptr, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *tmem_ptr;
  pdl_trigger();
  pdl_wait();                                        // the queries and the newest rows come from the previous kernels

  // warps: producer, MMA issuer, softmax groups, the other producers
  const int producer = warp == 0 ? 0 : warp - (2 + 4 * GROUPS) + 1;
  if (warp == 0 || warp >= 2 + 4 * GROUPS) {
    // ------------------------------------------------------------------ TMA producers
    const int* table = p.block_tables + static_cast<size_t>(b) * p.max_blocks;
    const uint64_t pol_q = l2_policy_evict_first(), pol_k = p.head_tiles > 1 ? l2_policy_evict_last() : l2_policy_evict_first();
    if (warp == 0 && lane == 0 && n_tiles > 0) {
      mbar_expect_tx(q_full, subs * Q_SUB);
      for (int c = 0; c < subs; ++c) tma_load_3d(q_sm + c * Q_SUB, &map_q, q_full, c * 64, b, h0, pol_q);
    }
    constexpr int BL = kLtKeys / kLtBlock;           // lanes 0-7: sub-tile lane / 4, pool block lane % 4
    const int last = (len - 1) / kLtBlock, total = n_tiles * np;
    const auto row_of = [&](int j) {                 // blocks past the sequence's end: the last one (masked)
      return lane < 2 * BL && j < n_tiles ? table[min((t0 + j) * BL + lane % BL, last)] * kLtBlock : 0;
    };
    int cur = producer / np, row = row_of(cur), next = row_of(cur + 1);
    for (int g = producer; g < total; g += kLtProducers) {   // this warp's slots
      const int j = g / np, i = g - j * np, slot = g % t.slots, ns = min(2, subs - 2 * i);
      while (cur < j) {                              // (the next tile's rows were asked for a tile ahead)
        row = next;
        next = row_of(++cur + 1);
      }
      bool ok = true;
      if (lane == 0) {
        ok = mbar_wait(&empty[slot], (static_cast<uint32_t>(g / t.slots) & 1u) ^ 1u, t.status, kErrLatentProducer);
        if (ok) mbar_expect_tx(&full[slot], ns * kLtSub);
      }
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
      if (!ok) break;
      if (lane < BL * ns)
        tma_load_2d(k_sm + slot * kLtSlot + (lane / BL) * kLtSub + (lane % BL) * (kLtBlock * 128), &map_pool, &full[slot],
                    (2 * i + lane / BL) * 64, row, pol_k);
      __syncwarp();
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    // The whole warp walks the schedule (so that its state stays in uniform registers: with N this small the issue rate
    // matters), one elected lane issues. The values of tile j - 1 go between the slots of tile j's scores: late enough
    // for their weights to be there, early enough to free their slots while the rest of tile j arrives.
    constexpr uint32_t idesc_s = umma_idesc_bf16(N, false, false, kLtKeys), idesc_o = umma_idesc_bf16(2 * N, true, false);
    const uint64_t ka = umma_desc_k_sw128(smem_u32(k_sm)), va = umma_desc_mn_sw128(smem_u32(k_sm), kLtSub, 1024),
                   qa = umma_desc_k_sw128(smem_u32(q_sm)), pa = umma_desc_k_sw128(smem_u32(p_sm));
    const bool elected = elect_one();
    int slot = 0, vs = 0;                            // next slot of the scores and of the values
    uint32_t phase = 0;
    bool ok = n_tiles == 0 || mbar_wait(q_full, 0, t.status, kErrLatentMma);
    const auto values = [&](int j) -> bool {
      if (!mbar_wait(&p_full[j & 1], static_cast<uint32_t>(j >> 1) & 1u, t.status, kErrLatentMma)) return false;
      tc_fence_after_sync();
      if (elected) {
        const uint64_t pj = pa + (j & 1) * (P_SUB >> 4);
        for (int m = 0, sl = vs; m < nm; ++m) {
          const uint64_t vm = va + sl * (kLtSlot >> 4);
#pragma unroll
          for (int kk = 0; kk < kLtKeys / 16; ++kk)
            umma_bf16(tmem + O_COL + m * 2 * N, vm + kk * (16 * 128 >> 4), pj + kk * 2, idesc_o, (j > 0 || kk > 0) ? 1u : 0u);
          umma_commit(&empty[sl]);
          if (++sl == t.slots) sl = 0;
        }
        umma_commit(&pv_done[j & 1]);
      }
      __syncwarp();
      vs += np;
      if (vs >= t.slots) vs -= t.slots;
      return true;
    };
    const int insert = np > 2 ? np - 2 : np - 1;     // the slot of tile j before which the values of tile j - 1 are issued
    const bool ahead = t.slots >= 2 * np;            // (a smaller ring: before its first slot)
    for (int j = 0; j < n_tiles && ok; ++j) {
      for (int i = 0; i < np; ++i) {
        if (j > 0 && i == (ahead ? insert : 0)) ok = values(j - 1);
        ok = ok && mbar_wait(&full[slot], phase, t.status, kErrLatentMma);
        if (!ok) break;
        tc_fence_after_sync();
        if (elected) {
          const uint64_t ks = ka + slot * (kLtSlot >> 4), qs = qa + i * (2 * Q_SUB >> 4);
          const uint32_t d = tmem + (j & 1) * 4 * N;
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) umma_bf16(d + kk * N, ks + kk * 2, qs + kk * 2, idesc_s, i > 0 ? 1u : 0u);
          if (2 * i + 1 < subs) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) umma_bf16(d + kk * N, ks + (kLtSub >> 4) + kk * 2, qs + (Q_SUB >> 4) + kk * 2, idesc_s, 1u);
          }
          if (i >= nm) umma_commit(&empty[slot]);    // no value columns in this slot
          if (i == np - 1) umma_commit(&s_full[j & 1]);
        }
        __syncwarp();
        if (++slot == t.slots) slot = 0, phase ^= 1u;
      }
    }
    if (ok && n_tiles > 0) values(n_tiles - 1);
  } else {
    // ------------------------------------------------------------------ softmax + epilogue
    const int q4 = warp & 3;                         // TMEM lanes a warp may touch: 32 (warp mod 4) ..
    const int key = q4 * 16 + (lane & 15);           // S row == token of the tile (lanes 16-31 hold none)
    const bool holds = lane < 16;
    const int g0 = ((warp - 2) >> 2) * HT;           // this thread's heads of the tile: g0 .. g0 + 15
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(q4 * 32) << 16) + g0;
    uint64_t* swap = &swap_bar[(warp - 2) >> 2];
    float* xm_all = reinterpret_cast<float*>(bars + 64) + 12 * g0;   // [2 buffers][4 warps][16]: maxima of a tile (a warp is
    float* xs = xm_all + 8 * HT;                                     // at most one exchange ahead); [4 warps][16]: sums
    float m_used[HT], l[HT];
#pragma unroll
    for (int n = 0; n < HT; ++n) m_used[n] = -INFINITY, l[n] = 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      ok = mbar_wait(&s_full[j & 1], static_cast<uint32_t>(j >> 1) & 1u, t.status, kErrLatentSoftmax);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after_sync();
      float sv[HT];
      {
        uint32_t r[4][HT];
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) tmem_ld_32x16(lane_addr + ((j & 1) * 4 + kk) * N, r[kk]);
        tmem_ld_wait();
        const int at = (t0 + j) * kLtKeys + key;
        const bool in = holds && at < len && at >= span.begin;
#pragma unroll
        for (int n = 0; n < HT; ++n) {
          const float s = (__uint_as_float(r[0][n]) + __uint_as_float(r[1][n])) + (__uint_as_float(r[2][n]) + __uint_as_float(r[3][n]));
          sv[n] = in ? s * p.scale_log2 : -INFINITY;
        }
      }
      float mine = -INFINITY;                        // lane n: this warp's maximum of head n
#pragma unroll
      for (int n = 0; n < HT; ++n) {
        const int x = __reduce_max_sync(0xffffffffu, float_order(__float_as_int(sv[n])));
        if (lane == n) mine = __int_as_float(float_order(x));
      }
      float* xm = xm_all + (j & 1) * 4 * HT;
      if (lane < HT) xm[q4 * HT + lane] = mine;
      __syncwarp();
      if (lane == 0) mbar_arrive(swap);
      ok = __all_sync(0xffffffffu, mbar_wait(swap, static_cast<uint32_t>(j) & 1u, t.status, kErrLatentSoftmax));
      if (!ok) break;
      bool rescale = false;
      float m_old[HT];
#pragma unroll
      for (int n = 0; n < HT; n += 4) {
        float4 a = *reinterpret_cast<const float4*>(xm + n);
#pragma unroll
        for (int w = 1; w < 4; ++w) {
          const float4 c = *reinterpret_cast<const float4*>(xm + w * HT + n);
          a.x = fmaxf(a.x, c.x), a.y = fmaxf(a.y, c.y), a.z = fmaxf(a.z, c.z), a.w = fmaxf(a.w, c.w);
        }
        const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float m = m_used[n + e];             // (the same in every thread; -inf + 8 stays below any score)
          m_old[n + e] = m;
          m_used[n + e] = av[e] > m + kLtRescale ? av[e] : m;
          rescale |= m_used[n + e] != m;
        }
      }
      if (j > 1) {                                   // the weight buffer belongs to the values of tile j - 2 until they are through
        ok = __all_sync(0xffffffffu, mbar_wait(&pv_done[j & 1], static_cast<uint32_t>((j - 2) >> 1) & 1u, t.status, kErrLatentSoftmax));
        if (!ok) break;
      }
      if (rescale && j > 0) {                        // O is at rest once the values of tile j - 1 are through
        ok = __all_sync(0xffffffffu, mbar_wait(&pv_done[(j - 1) & 1], static_cast<uint32_t>((j - 1) >> 1) & 1u, t.status, kErrLatentSoftmax));
        if (!ok) break;
        tc_fence_after_sync();
        float alpha[HT];
#pragma unroll
        for (int n = 0; n < HT; ++n) alpha[n] = exp2f(m_old[n] - m_used[n]);
        for (int m = 0; m < 2 * nm; ++m) {           // both terms' sums
          uint32_t r[HT];
          tmem_ld_32x16(lane_addr + O_COL + m * N, r);
          tmem_ld_wait();
#pragma unroll
          for (int n = 0; n < HT; ++n) r[n] = __float_as_uint(__uint_as_float(r[n]) * alpha[n]);
          tmem_st_32x16(lane_addr + O_COL + m * N, r);
        }
        tmem_st_wait();
#pragma unroll
        for (int n = 0; n < HT; ++n) l[n] *= alpha[n];
      }
      // weights, two tokens per 32-bit store: the even lane of a pair stores the even head, the odd lane the odd one
      uint8_t* prow = p_sm + (j & 1) * P_SUB + g0 * 128;
      const uint32_t pcol = static_cast<uint32_t>(key & 6) * 2, chunk = static_cast<uint32_t>(key) >> 3;
      const bool odd = lane & 1;
#pragma unroll
      for (int n = 0; n < HT; n += 2) {
        const float e0 = exp2f(sv[n] - m_used[n]), e1 = exp2f(sv[n + 1] - m_used[n + 1]);
        l[n] += e0, l[n + 1] += e1;
        const float got = __shfl_xor_sync(0xffffffffu, odd ? e0 : e1, 1);
        const float lo = odd ? got : e0, hi = odd ? e1 : got;
        const int row = n + (odd ? 1 : 0);
        const uint32_t pk = pack_bf16(lo, hi), rest = pack_bf16(lo - bf16_lo(pk), hi - bf16_hi(pk));
        uint8_t* dst = prow + row * 128 + ((chunk ^ (row & 7)) << 4) + pcol;
        if (holds) {
          *reinterpret_cast<uint32_t*>(dst) = pk;
          *reinterpret_cast<uint32_t*>(dst + N * 128) = rest;
        }
      }
      fence_proxy_async_smem();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[j & 1]);
    }
    // ---- this split's sums, then one latent column per thread
    const int heads = min(HT, p.H - h0 - g0);        // (may be negative)
    if (ok) {
#pragma unroll
      for (int n = 0; n < HT; ++n) {
        const float s = warp_sum(l[n]);
        if (lane == n) xs[q4 * HT + n] = s;
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(swap);
      ok = mbar_wait(swap, static_cast<uint32_t>(n_tiles) & 1u, t.status, kErrLatentSoftmax);
      for (int j = max(0, n_tiles - 2); ok && j < n_tiles; ++j)
        ok = mbar_wait(&pv_done[j & 1], static_cast<uint32_t>(j >> 1) & 1u, t.status, kErrLatentSoftmax);
    }
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tc_fence_after_sync();
      const size_t part = static_cast<size_t>(bt) * p.num_splits + split;
      if (p.num_splits > 1 && q4 == 0) {
#pragma unroll
        for (int n = 0; n < HT; ++n) {
          if (lane == n) {
            p.scratch_ml[(part * N + g0 + n) * 2] = m_used[n];
            p.scratch_ml[(part * N + g0 + n) * 2 + 1] = xs[n] + xs[HT + n] + xs[2 * HT + n] + xs[3 * HT + n];
          }
        }
      }
      if (n_tiles > 0 || p.num_splits == 1) {        // (a split without tokens leaves its weights' sum 0: never read)
        for (int m = 0; m < nm; ++m) {
          float o[HT];
#pragma unroll
          for (int n = 0; n < HT; ++n) o[n] = 0.f;
          if (n_tiles > 0) {
            uint32_t r[HT], r2[HT];
            tmem_ld_32x16(lane_addr + O_COL + m * 2 * N, r);
            tmem_ld_32x16(lane_addr + O_COL + m * 2 * N + N, r2);
            tmem_ld_wait();
#pragma unroll
            for (int n = 0; n < HT; ++n) o[n] = __uint_as_float(r[n]) + __uint_as_float(r2[n]);
          }
          const int c = m * 128 + q4 * 32 + lane;    // O row == TMEM lane
          if (c < p.C) {
#pragma unroll
            for (int n = 0; n < HT; ++n) {
              if (n >= heads) break;
              if (p.num_splits > 1) {
                p.scratch_o[(part * N + g0 + n) * p.C + c] = o[n];
              } else {
                float f;
                const float s = latent_denominator(p, h0 + g0 + n, m_used[n], xs[n] + xs[HT + n] + xs[2 * HT + n] + xs[3 * HT + n], f);
                p.out[(static_cast<size_t>(b) * p.H + h0 + g0 + n) * p.C + c] = __float2bfloat16(s > 0.f ? o[n] * f / s : 0.f);
              }
            }
          }
        }
      }
    }
  }
  // ------------------------------------------------------------------ teardown
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, TMEM_COLS);
  }
}

template <int N>
static int launch_latent_tc(const CUtensorMap& mq, const CUtensorMap& mp, LatentTcParams t, int grid, cudaStream_t st) {
  constexpr int limit = 227 * 1024;
  const int np = (t.d.W + 127) / 128, fixed = lt_fixed_smem(t.d.W, N);
  int slots = (limit - fixed) / kLtSlot;
  if (slots > kLtMaxSlots) slots = kLtMaxSlots;
  if (slots < np) return -10;
  t.slots = slots > 4 * np ? 4 * np : slots;
  auto kern = latent_decode_tc_kernel<N>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, limit);
    if (e != cudaSuccess) return static_cast<int>(e);
    prefer_max_shared(kern);
    configured = true;
  }
  return static_cast<int>(launch_kernel(kern, dim3(grid), dim3(lt_threads(N)), fixed + t.slots * kLtSlot, st, mq, mp, t));
}

int latent_decode_tc(const LatentDecodeParams& d, int B, long long pool_rows, int* status, cudaStream_t st) {
  if (d.block_size != kLtBlock || status == nullptr || pool_rows <= 0 || (d.head_tile != 16 && d.head_tile != 32)) return -10;
  CUtensorMap mq, mp;
  if (!make_tensor_map_bf16_3d(&mq, d.q, d.H, B, d.W, d.W, d.q_stride, d.head_tile, 64) ||
      !make_tensor_map_bf16(&mp, d.pool, pool_rows, d.W, d.W, kLtBlock, 64))
    return -4;
  LatentTcParams t{d, status, 0};
  const int grid = B * d.head_tiles * d.num_splits;
  return d.head_tile == 32 ? launch_latent_tc<32>(mq, mp, t, grid, st) : launch_latent_tc<16>(mq, mp, t, grid, st);
}

}  // namespace mx
