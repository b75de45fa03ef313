// Chunked causal prefill attention on the 5th-generation tensor cores (tcgen05 + TMEM + TMA).
//
// A CTA owns 128 consecutive query tokens of one query head and walks the visible keys of the
// paged KV pool in tiles of 128 keys (8 pool blocks of 16):
//
//   warp 0     TMA producer: Q once; per KV tile the eight K and eight V block slabs of the pool
//              (each [16 keys][D] bf16, contiguous per (block, kv head)) land as 128-byte-swizzled
//              shared-memory tiles, lanes 0-7 issuing one block each
//   warp 1     MMA issuer: S = Q K^T (M=128, N=128, K=D) into one of two TMEM score buffers, then
//              O += P V (M=128, N=D, K=128 keys) with P read from shared memory and V consumed
//              MN-major, exactly as it sits in the pool
//   warps 2-5  (2-9 in the extended form) softmax, one (two) threads per query row: tcgen05.ld the scores, mask, running max with
//              lazy rescaling (O in TMEM is rescaled only when a row maximum grows by more than
//              2^8, the final normalisation uses the same stale maximum, so the result is exact),
//              P = exp2(...) written as the bf16 A operand of the next MMA, and the epilogue
//
// S is double-buffered, so the score MMA of tile j+1 runs while the softmax of tile j does.
// Every wait is bounded and reports through the status word.
//
// Replaces the reference's cuDNN SDPA prefill (mlx/backend/cuda/scaled_dot_product_attention.cpp in
// its MLX overlay) and `chunked_causal_attention` (src/lib/mlxcel-core/src/layers.rs:5798).
#include "api.h"
#include "common.cuh"

namespace mx {

bool make_tensor_map_bf16(CUtensorMap* out, const void* ptr, uint64_t rows, uint64_t cols,
                          uint64_t ld, uint32_t box_rows, uint32_t box_cols);
bool make_tensor_map_bf16_3d(CUtensorMap* out, const void* ptr, uint64_t rows, uint64_t groups, uint64_t cols, uint64_t ld,
                             uint64_t group_ld, uint32_t box_rows, uint32_t box_cols);

constexpr int kTcRows = 128;      // query rows per CTA (UMMA M)
constexpr int kTcKeys = 128;      // keys per tile
constexpr int kTcStages = 2;
constexpr int kTcBlock = 16;      // pool block size this kernel is written for
constexpr float kRescaleThreshold = 8.0f;   // log2 units

enum : int { kErrAttnProducer = 401, kErrAttnMma = 402, kErrAttnSoftmax = 403 };

struct TcPrefillParams {
  const int* block_tables;
  const int* cu_q;
  const int* context_lens;
  const float* sinks;
  __nv_bfloat16* out;
  int* status;
  int num_seqs, Hq, Hkv, max_blocks, window, tiles_per_seq;
  float scale_log2;
  // Extended form (EXT): rows of dk / dv elements inside tiles of DK / DV columns (the tensor maps end at
  // the row's width, so the missing columns arrive as zeros), a logarithmic distance bias
  // r1[h] ln(1 + r2[h] d) taken off the scores, an output gate (result *= sigmoid(gate)); bias and gate
  // may be NULL. chunk > 0: keys of the query's own run of `chunk` positions only; softcap > 0: scores s become
  // softcap tanh(s / softcap).
  int dk, dv, chunk;
  float softcap;
  const float* bias_r1;
  const float* bias_r2;
  const __nv_bfloat16* gate;
  long long gate_stride;
  // Dense keys and values (kv_starts != NULL, no pool): the context of sequence s lies in rows kv_starts[s] .. of
  // per-head key and value matrices, and the key's last columns (from kv_split on, one 64-column tile) come from
  // a matrix all heads share.
  const int* kv_starts;
  int kv_split;
  long long out_stride;      // elements between output rows
  // Differential heads (MAPS == 2): the result is (a1 - lambda a2) / rms(.) * gain. With one map, gain is a plain factor
  // of the extended form's result.
  float lambda, gain, eps;
  // Block means (MEANS, with a window): beside the window's tokens, one key and value for every block of mean_of tokens
  // wholly before the window, gathered to dense rows: block b of sequence s is row mean_starts[s] + b.
  const int* mean_starts;
  int mean_of;
};

// The extended form runs eight softmax warps instead of four, two per 32 query rows: each takes one half of
// a tile's keys (and of the output columns), the two exchange their row maxima once per tile and their sums
// at the end through shared memory, under an mbarrier with the usual bounded wait.
__host__ __device__ constexpr int tc_softmax_warps(bool ext) { return ext ? 8 : 4; }
__host__ __device__ constexpr int tc_threads(bool ext) { return 64 + 32 * tc_softmax_warps(ext); }

// Distances between a warp's 32 query rows and its 64 keys of a tile take 95 values: it tabulates their biases
// once per tile instead of taking a logarithm per score.
constexpr int kBiasTab = 96;
constexpr int kExtSmem = 8 * kBiasTab * 4 + 2 * 2 * kTcRows * 4 + 2 * kTcRows * 4;   // tables, maxima (2 buffers), sums

// Differential heads (MAPS == 2, no sinks, bias or gate): query and key heads are two maps of dk columns each. The CTA walks
// its key tiles twice, first with map 1, then with map 2 (tile j of the walk is key tile j mod n of map j / n), with running
// maxima and sums per map and an accumulator each in TMEM; the epilogue combines the two in registers. Scores of map
// 2's first tile run under the softmax of map 1's last one, as between any two tiles.
//
// Block means (MEANS): the walk begins with the tiles of 128 means that some query of the CTA sees, then the window's tokens. Rows of
// a means' tile past a query's last visible block are masked (they belong to later blocks, the next sequence, or are zero).
//
// The second weight term takes the room of one V stage where both heads are 128 wide: a V tile is only
// needed once its softmax is through, so its load still has most of a tile's time.
__host__ __device__ constexpr int tc_v_stages(int dk, int dv, bool ext) { return (ext && dk >= 128 && dv == 128) ? 1 : kTcStages; }
// Keys of 192 columns (and two maps of queries of 128) leave room for one K stage (free again as soon as its score MMA has run).
__host__ __device__ constexpr int tc_k_stages(int dk, int maps) { return dk > 128 || (dk == 128 && maps == 2) ? 1 : kTcStages; }

template <int DK, int DV, bool EXT, int MAPS, bool MEANS>
__global__ void __launch_bounds__(tc_threads(EXT), 1)
paged_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                        const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_kr,
                        const __grid_constant__ CUtensorMap map_vm, const TcPrefillParams p) {
  // (map_kr: the shared key part of dense rows, or the means' keys; map_vm: the means' values)
  constexpr int DC = DK / 64, DCV = DV / 64;          // 64-column (128-byte) sub-tiles per row
  constexpr int SUB_BYTES = 128 * 128;                // one [128 rows][64 cols] sub-tile
  constexpr int Q_BYTES = DC * SUB_BYTES;
  constexpr int K_BYTES = DC * SUB_BYTES;             // [128 keys][DK]
  constexpr int V_BYTES = DCV * SUB_BYTES;
  constexpr int PHALF_BYTES = 2 * SUB_BYTES;          // [128 rows][128 keys]
  // The extended form feeds the weights to the second product as a sum of two bf16 terms (the rounded
  // weight and what the rounding left), which keeps 16 bits of each: two MMAs per step instead of one.
  constexpr int PTERMS = EXT ? 2 : 1;
  constexpr int P_BYTES = PTERMS * PHALF_BYTES;
  constexpr int VST = tc_v_stages(DK, DV, EXT);       // V ring depth
  constexpr int KST = tc_k_stages(DK, MAPS);          // K ring depth
  constexpr int S_COLS = kTcKeys;                     // fp32 columns of one score buffer
  constexpr int O_COL = 2 * S_COLS;                   // first TMEM column of O (DV columns per map)
  constexpr uint32_t TMEM_COLS = 512;
  static_assert((DK == 64 || DK == 128 || (EXT && DK == 192)) && (DV == 64 || DV == 128), "head dims");
  static_assert(EXT || DK == DV, "plain form: one head width");
  static_assert(MAPS == 1 || EXT, "differential heads: extended form");
  static_assert(!MEANS || (EXT && MAPS == 1), "block means: extended form, one map");
  const int dk = EXT ? p.dk : DK, dv = EXT ? p.dv : DV;

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  uint8_t* q_sm = smem;
  uint8_t* k_sm = q_sm + MAPS * Q_BYTES;              // KST x K_BYTES
  uint8_t* v_sm = k_sm + KST * K_BYTES;               // VST x V_BYTES
  uint8_t* p_sm = v_sm + VST * V_BYTES;
  uint64_t* bars = reinterpret_cast<uint64_t*>(p_sm + P_BYTES);
  uint64_t* q_full = bars;                // 1
  uint64_t* k_full = bars + 1;            // [stages]
  uint64_t* v_full = k_full + kTcStages;  // [stages]
  uint64_t* kv_empty = v_full + kTcStages;   // [stages]
  uint64_t* s_full = kv_empty + kTcStages;   // [2]
  uint64_t* s_empty = s_full + 2;            // [2]
  uint64_t* p_full = s_empty + 2;            // 1
  uint64_t* pv_done = p_full + 1;            // 1
  uint64_t* k_empty = pv_done + 1;           // [stages] K tile consumed (after the score MMA)
  uint64_t* pair_bar = k_empty + kTcStages;  // [4] EXT: the two warps of 32 rows exchange
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(pair_bar + 4);
  float* bias_tab = reinterpret_cast<float*>(p_sm + P_BYTES + 256);   // EXT: 8 warps x kBiasTab
  float* pair_max = bias_tab + 8 * kBiasTab;                          // EXT: [2 buffers][2 halves][128 rows]
  float* pair_sum = pair_max + 4 * kTcRows;                           // EXT: [2 halves][128 rows]
  constexpr int SWARPS = tc_softmax_warps(EXT), HALVES = SWARPS / 4;
  constexpr int HC = kTcKeys / HALVES;                                // key columns per softmax thread

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  // ---- which tile (heavy tiles, i.e. late tokens, first)
  const int tile = p.tiles_per_seq - 1 - static_cast<int>(blockIdx.x % p.tiles_per_seq);
  const int sh = blockIdx.x / p.tiles_per_seq;
  const int hq = sh % p.Hq, s = sh / p.Hq;
  const int hkv = hq / (p.Hq / p.Hkv);
  const int q0 = p.cu_q[s], q_len = p.cu_q[s + 1] - q0;
  const int tok0 = tile * kTcRows;
  if (tok0 >= q_len) return;   // whole CTA leaves before any barrier / TMEM use
  const int ctx = p.context_lens[s];
  const int pos_base = ctx - q_len;   // absolute position of query token 0
  const int rows_valid = min(kTcRows, q_len - tok0);
  const int kv_end = pos_base + tok0 + rows_valid;   // one past the last visible key
  int kv_begin = 0;
  if (p.window > 0) kv_begin = max(0, pos_base + tok0 - p.window + 1);
  if constexpr (EXT) {
    if (p.chunk > 0) kv_begin = max(kv_begin, (pos_base + tok0) / p.chunk * p.chunk);
  }
  kv_begin = (kv_begin / kTcKeys) * kTcKeys;
  const int key_tiles = (kv_end - kv_begin + kTcKeys - 1) / kTcKeys;
  // (the last query of the tile sees the most means)
  const int mean_tiles = MEANS ? (max(0, kv_end - p.window) / p.mean_of + kTcKeys - 1) / kTcKeys : 0;
  const int n_tiles = MAPS * key_tiles + mean_tiles;  // tiles of the walk
  const auto key_tile = [&](int j) { return MAPS == 2 && j >= key_tiles ? j - key_tiles : j - mean_tiles; };
  const auto map_of = [&](int j) { return MAPS == 2 && j >= key_tiles ? 1 : 0; };
  const int last_block = (ctx - 1) / kTcBlock;   // last pool block the sequence owns

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_k);
    tma_prefetch_desc(&map_v);
    mbar_init(q_full, 1);
    for (int i = 0; i < kTcStages; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&kv_empty[i], 1);
      mbar_init(&k_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], SWARPS);
    }
    mbar_init(p_full, SWARPS);
    for (int i = 0; i < 4; ++i) mbar_init(&pair_bar[i], 2);
    mbar_init(pv_done, 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_ptr, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_ptr;
  pdl_trigger();
  pdl_wait();   // q and the newest keys come from the previous kernels of the step

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    const int* table = p.block_tables + static_cast<size_t>(s) * p.max_blocks;
    const uint64_t pol_q = l2_policy_evict_first();
    const uint64_t pol_kv = l2_policy_evict_last();   // re-read by the other heads / token tiles
    if (lane == 0) {
      mbar_expect_tx(q_full, MAPS * Q_BYTES);
      for (int c = 0; c < MAPS * DC; ++c)
        if (MAPS == 2)
          tma_load_3d(q_sm + c * SUB_BYTES, &map_q, q_full, (c % DC) * 64, hq * 2 + c / DC, q0 + tok0, pol_q);
        else if (EXT && p.kv_starts != nullptr)
          tma_load_3d(q_sm + c * SUB_BYTES, &map_q, q_full, c * 64 < p.kv_split ? c * 64 : p.kv_split, hq, q0 + tok0, pol_q);
        else
          tma_load_2d(q_sm + c * SUB_BYTES, &map_q, q_full, hq * dk + c * 64, q0 + tok0, pol_q);
    }
    int stage = 0;
    uint32_t phase = 0;
    bool ok = true;
    if (EXT && MAPS == 1 && p.kv_starts != nullptr) {
      // dense rows: one box per 64-column tile (rows past the sequence belong to the next one or are filled with
      // zeros; the mask drops them)
      const int base = p.kv_starts[s];
      for (int j = 0; lane == 0 && j < n_tiles; ++j) {
        const int row0 = base + kv_begin + j * kTcKeys, ks = j % KST, vs = j % VST;
        if (!mbar_wait(&k_empty[ks], (static_cast<uint32_t>(j / KST) & 1u) ^ 1u, p.status, kErrAttnProducer)) break;
        mbar_expect_tx(&k_full[ks], K_BYTES);
        for (int c = 0; c < DC; ++c) {
          uint8_t* kd = k_sm + ks * K_BYTES + c * SUB_BYTES;
          if (c * 64 < p.kv_split) tma_load_3d(kd, &map_k, &k_full[ks], c * 64, hkv, row0, pol_kv);
          else tma_load_2d(kd, &map_kr, &k_full[ks], 0, row0, pol_kv);
        }
        if (!mbar_wait(&kv_empty[vs], (static_cast<uint32_t>(j / VST) & 1u) ^ 1u, p.status, kErrAttnProducer)) break;
        mbar_expect_tx(&v_full[vs], V_BYTES);
        for (int c = 0; c < DCV; ++c) tma_load_3d(v_sm + vs * V_BYTES + c * SUB_BYTES, &map_v, &v_full[vs], c * 64, hkv, row0, pol_kv);
      }
      ok = false;
    }
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int vstage = j % VST;
      const uint32_t vphase = static_cast<uint32_t>(j / VST) & 1u;
      // The K tile of a stage is free as soon as its score MMA has run, the V tile only after the
      // P V MMA of the same key tile: K of tile j + stages is requested a whole softmax earlier.
      // one pool block per lane; blocks past the sequence's last one repeat it (masked keys, but
      // the values multiplied by P = 0 must be finite)
      if (MEANS && j < mean_tiles) {
        // a tile of means: one box per 64-column sub-tile
        if (lane == 0) {
          const int m0 = p.mean_starts[s] + j * kTcKeys;
          ok = mbar_wait(&k_empty[stage], phase ^ 1u, p.status, kErrAttnProducer);
          if (ok) {
            mbar_expect_tx(&k_full[stage], K_BYTES);
            for (int c = 0; c < DC; ++c) tma_load_3d(k_sm + stage * K_BYTES + c * SUB_BYTES, &map_kr, &k_full[stage], c * 64, hkv, m0, pol_kv);
            ok = mbar_wait(&kv_empty[vstage], vphase ^ 1u, p.status, kErrAttnProducer);
          }
          if (ok) {
            mbar_expect_tx(&v_full[vstage], V_BYTES);
            for (int c = 0; c < DCV; ++c) tma_load_3d(v_sm + vstage * V_BYTES + c * SUB_BYTES, &map_vm, &v_full[vstage], c * 64, hkv, m0, pol_kv);
          }
        }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (++stage == KST) {
          stage = 0;
          phase ^= 1u;
        }
        continue;
      }
      int row0 = 0;
      if (lane < kTcKeys / kTcBlock) {
        const int b = min((kv_begin + key_tile(j) * kTcKeys) / kTcBlock + lane, last_block);
        row0 = (table[b] * p.Hkv + hkv) * kTcBlock;
      }
      if (lane == 0) {
        ok = mbar_wait(&k_empty[stage], phase ^ 1u, p.status, kErrAttnProducer);
        if (ok) mbar_expect_tx(&k_full[stage], K_BYTES);
      }
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
      if (!ok) break;
      if (lane < kTcKeys / kTcBlock) {
        uint8_t* kd = k_sm + stage * K_BYTES + lane * (kTcBlock * 128);
        for (int c = 0; c < DC; ++c) {
          if (MAPS == 2) tma_load_3d(kd + c * SUB_BYTES, &map_k, &k_full[stage], c * 64, map_of(j), row0, pol_kv);
          else tma_load_2d(kd + c * SUB_BYTES, &map_k, &k_full[stage], c * 64, row0, pol_kv);
        }
      }
      if (lane == 0) {
        ok = mbar_wait(&kv_empty[vstage], vphase ^ 1u, p.status, kErrAttnProducer);
        if (ok) mbar_expect_tx(&v_full[vstage], V_BYTES);
      }
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
      if (!ok) break;
      if (lane < kTcKeys / kTcBlock) {
        uint8_t* vd = v_sm + vstage * V_BYTES + lane * (kTcBlock * 128);
        for (int c = 0; c < DCV; ++c) tma_load_2d(vd + c * SUB_BYTES, &map_v, &v_full[vstage], c * 64, row0, pol_kv);
      }
      __syncwarp();
      if (++stage == KST) {
        stage = 0;
        phase ^= 1u;
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_qk = umma_idesc_bf16(kTcKeys, false, false);   // N = keys
      constexpr uint32_t idesc_pv = umma_idesc_bf16(DV, false, true);         // N = DV, V is MN-major
      bool ok = mbar_wait(q_full, 0, p.status, kErrAttnMma);
      auto issue_qk = [&](int j) -> bool {
        const int stage = j % KST;
        const uint32_t kv_phase = static_cast<uint32_t>(j / KST) & 1u;
        const int sb = j & 1;
        const uint32_t s_phase = static_cast<uint32_t>(j >> 1) & 1u;
        if (!mbar_wait(&k_full[stage], kv_phase, p.status, kErrAttnMma)) return false;
        if (!mbar_wait(&s_empty[sb], s_phase ^ 1u, p.status, kErrAttnMma)) return false;
        tc_fence_after_sync();
        const uint32_t qa = smem_u32(q_sm) + map_of(j) * Q_BYTES, kb = smem_u32(k_sm + stage * K_BYTES);
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const uint32_t off = (kk >> 2) * SUB_BYTES + (kk & 3) * 32;
          umma_bf16(tmem_base + sb * S_COLS, umma_desc_k_sw128(qa + off), umma_desc_k_sw128(kb + off),
                    idesc_qk, kk > 0 ? 1u : 0u);
        }
        umma_commit(&k_empty[stage]);   // the K tile may be refilled
        umma_commit(&s_full[sb]);
        return true;
      };
      if (ok) ok = issue_qk(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (j + 1 < n_tiles) ok = issue_qk(j + 1);   // scores of the next tile under this softmax
        if (!ok) break;
        const int stage = j % VST;
        const uint32_t v_phase = static_cast<uint32_t>(j / VST) & 1u;
        if (!mbar_wait(&v_full[stage], v_phase, p.status, kErrAttnMma)) break;
        if (!mbar_wait(p_full, static_cast<uint32_t>(j) & 1u, p.status, kErrAttnMma)) break;
        tc_fence_after_sync();
        const uint32_t pa = smem_u32(p_sm), vb = smem_u32(v_sm + stage * V_BYTES);
#pragma unroll
        for (int kk = 0; kk < kTcKeys / 16; ++kk) {
          const uint64_t db = umma_desc_mn_sw128(vb + kk * (16 * 128), SUB_BYTES, 1024);
#pragma unroll
          for (int term = 0; term < PTERMS; ++term) {
            const uint64_t da = umma_desc_k_sw128(pa + term * PHALF_BYTES + (kk >> 2) * SUB_BYTES + (kk & 3) * 32);
            umma_bf16(tmem_base + O_COL + map_of(j) * DV, da, db, idesc_pv, ((MEANS ? j : key_tile(j)) > 0 || kk > 0 || term > 0) ? 1u : 0u);
          }
        }
        umma_commit(&kv_empty[stage]);   // the V tile of this stage is consumed
        umma_commit(pv_done);
      }
    }
    __syncwarp();
  } else {
    // ------------------------------------------------------------------ softmax + epilogue
    const int q4 = warp & 3;                        // TMEM lanes a warp may touch: 32 (warp mod 4) ..
    const int half = HALVES == 2 ? (warp - 2) >> 2 : 0;   // EXT: keys half * 64 .. + 63 of every tile
    const int row = q4 * 32 + lane;                 // query row == TMEM lane
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(q4 * 32) << 16);
    const int qpos = pos_base + tok0 + row;         // absolute position of this row's token
    float m_used = -INFINITY;   // the maximum the stored exponentials refer to (scaled, log2 units)
    float l = 0.f, l_first = 0.f;                   // (MAPS == 2: the first map's sum)
    float* tab = bias_tab + (warp - 2) * kBiasTab;
    float r1 = 0.f, r2 = 0.f;
    const __nv_bfloat16* gate = nullptr;            // this row's gate values, needed in the epilogue
    if constexpr (EXT) {
      if (p.bias_r1 != nullptr) r1 = p.bias_r1[hq], r2 = p.bias_r2[hq];
      if (p.gate != nullptr && row < rows_valid) {
        gate = p.gate + static_cast<size_t>(q0 + tok0 + row) * p.gate_stride + hq * dv;
        for (int i = 0; i < dv; i += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(gate + i));
      }
    }
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int sb = j & 1;
      const uint32_t s_phase = static_cast<uint32_t>(j >> 1) & 1u;
      if (MAPS == 2 && j == key_tiles) {
        l_first = l;
        l = 0.f;
        m_used = -INFINITY;
      }
      ok = mbar_wait(&s_full[sb], s_phase, p.status, kErrAttnSoftmax);
      if (!ok) break;
      tc_fence_after_sync();
      const int o_col = O_COL + map_of(j) * DV;
      const bool mean = MEANS && j < mean_tiles;
      const int key0 = mean ? j * kTcKeys : kv_begin + key_tile(j) * kTcKeys;      // (of a tile of means: its first block)
      // Only tiles that cross the diagonal, the window edge or the end need the mask.
      const bool need_mask = (key0 + kTcKeys - 1 > pos_base + tok0) ||
                             (p.window > 0 && key0 < pos_base + tok0 + kTcRows - p.window) ||
                             (EXT && p.chunk > 0 && key0 < (pos_base + tok0 + rows_valid - 1) / p.chunk * p.chunk);
      const int hkey0 = key0 + half * HC;   // first key of this thread's columns
      int lo = 0, hi = HC;   // valid key columns of this row: [lo, hi)
      if (mean) {
        hi = min(HC, max(0, qpos + 1 - p.window) / p.mean_of - hkey0);
      } else if (need_mask) {
        hi = min(HC, qpos - hkey0 + 1);
        if (p.window > 0) lo = max(0, qpos - p.window + 1 - hkey0);
        if (EXT && p.chunk > 0) lo = max(lo, qpos / p.chunk * p.chunk - hkey0);
      }
      if (EXT && p.bias_r1 != nullptr) {
        // tab[i] = bias of distance base + i, where row r of this warp and key column c are at
        // i = r - c + 63 (log2 domain: the natural logarithm's factor cancels against log2 e)
        const int base = pos_base + tok0 + q4 * 32 - hkey0 - (HC - 1);
        __syncwarp();
#pragma unroll
        for (int i = 0; i < kBiasTab / 32; ++i) {
          const float d = static_cast<float>(max(base + lane + i * 32, 0));
          tab[lane + i * 32] = r1 * log2f(fmaf(r2, d, 1.f));
        }
        __syncwarp();
      }
      float sv[HC];
#pragma unroll
      for (int c = 0; c < HC / 32; ++c) {
        uint32_t r[32];
        tmem_ld_32x32(lane_addr + sb * S_COLS + half * HC + c * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          sv[c * 32 + i] = __uint_as_float(r[i]) * p.scale_log2;
        }
        if constexpr (EXT) {
          if (p.softcap > 0.f) {
#pragma unroll
            for (int i = 0; i < 32; ++i) sv[c * 32 + i] = soft_cap_log2(sv[c * 32 + i], p.softcap);
          }
          if (p.bias_r1 != nullptr) {
#pragma unroll
            for (int i = 0; i < 32; ++i) sv[c * 32 + i] -= tab[lane + (HC - 1) - (c * 32 + i)];
          }
        }
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_empty[sb]);   // the score buffer may be overwritten
      float mx = -INFINITY;
      if (need_mask || mean) {
#pragma unroll
        for (int i = 0; i < HC; ++i) {
          if (i < lo || i >= hi) sv[i] = -INFINITY;
          mx = fmaxf(mx, sv[i]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < HC; ++i) mx = fmaxf(mx, sv[i]);
      }
      if constexpr (HALVES == 2) {
        // the row's maximum over both halves (two buffers: a warp is at most one exchange ahead)
        float* xm = pair_max + (j & 1) * 2 * kTcRows;
        xm[half * kTcRows + row] = mx;
        __syncwarp();
        if (lane == 0) mbar_arrive(&pair_bar[q4]);
        ok = mbar_wait(&pair_bar[q4], static_cast<uint32_t>(j) & 1u, p.status, kErrAttnSoftmax);
        if (!ok) break;
        mx = fmaxf(mx, xm[(half ^ 1) * kTcRows + row]);
      }
      // lazy rescaling: keep the old reference maximum unless the row grew past it by 2^8
      float alpha = 1.0f;
      bool rescale = false;
      if (mx > m_used + kRescaleThreshold || m_used == -INFINITY) {
        if (mx > -INFINITY) {
          alpha = (m_used == -INFINITY) ? 0.0f : exp2f(m_used - mx);
          rescale = (m_used != -INFINITY);
          m_used = mx;
        }
      }
      // O and the P buffer belong to the previous tile's P V until that MMA has finished.
      if (j > 0) {
        ok = mbar_wait(pv_done, static_cast<uint32_t>(j - 1) & 1u, p.status, kErrAttnSoftmax);
        if (!ok) break;
        tc_fence_after_sync();
      }
      if (__any_sync(0xffffffffu, rescale)) {
#pragma unroll
        for (int cc = 0; cc < DV / 32 / HALVES; ++cc) {
          const int c = half * (DV / 32 / HALVES) + cc;
          uint32_t r[32];
          tmem_ld_32x32(lane_addr + o_col + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
          tmem_st_32x32(lane_addr + o_col + c * 32, r);
        }
        tmem_st_wait();
      }
      l *= alpha;
      // P = exp2(s - m) as bf16, K-major with the 128-byte swizzle (row = query, 16-byte chunk
      // index XOR (row & 7) inside each 64-key sub-tile)
      float sum = 0.f;
      const float mref = (m_used == -INFINITY) ? 0.f : m_used;
#pragma unroll
      for (int c8 = 0; c8 < HC / 8; ++c8) {
        float e[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          e[i] = exp2f(sv[c8 * 8 + i] - mref);   // exp2(-inf) = 0 for masked keys
          sum += e[i];
        }
        uint4 pk;
        pk.x = pack_bf16(e[0], e[1]);
        pk.y = pack_bf16(e[2], e[3]);
        pk.z = pack_bf16(e[4], e[5]);
        pk.w = pack_bf16(e[6], e[7]);
        const int sub = half + (c8 >> 3), ch = c8 & 7;
        uint8_t* pd = p_sm + sub * SUB_BYTES + row * 128 + ((ch ^ (row & 7)) << 4);
        *reinterpret_cast<uint4*>(pd) = pk;
        if constexpr (EXT) {
          uint4 rk;
          rk.x = pack_bf16(e[0] - bf16_lo(pk.x), e[1] - bf16_hi(pk.x));
          rk.y = pack_bf16(e[2] - bf16_lo(pk.y), e[3] - bf16_hi(pk.y));
          rk.z = pack_bf16(e[4] - bf16_lo(pk.z), e[5] - bf16_hi(pk.z));
          rk.w = pack_bf16(e[6] - bf16_lo(pk.w), e[7] - bf16_hi(pk.w));
          *reinterpret_cast<uint4*>(pd + PHALF_BYTES) = rk;
        }
      }
      l += sum;
      fence_proxy_async_smem();   // generic-proxy writes of P -> visible to the MMA's async proxy
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    // ---- epilogue: O / l -> out (one row of D bf16 per thread; EXT: half a row)
    if constexpr (MAPS == 2) {
      // sums of both maps over the two halves, then the combined row: its square sum takes one more exchange
      constexpr int CW = DV / 2;                    // columns of a thread
      float inv1 = 0.f, inv2 = 0.f, av[CW];
      if (ok) {
        pair_sum[half * kTcRows + row] = l;
        pair_max[half * kTcRows + row] = l_first;   // (the maxima of the tiles before the last are through: see below)
        __syncwarp();
        if (lane == 0) mbar_arrive(&pair_bar[q4]);
        ok = mbar_wait(&pair_bar[q4], static_cast<uint32_t>(n_tiles) & 1u, p.status, kErrAttnSoftmax);
        const float l1 = pair_max[row] + pair_max[kTcRows + row], l2 = pair_sum[row] + pair_sum[kTcRows + row];
        inv1 = l1 > 0.f ? 1.f / l1 : 0.f;
        inv2 = l2 > 0.f ? p.lambda / l2 : 0.f;
      }
      if (ok) ok = mbar_wait(pv_done, static_cast<uint32_t>(n_tiles - 1) & 1u, p.status, kErrAttnSoftmax);
      if (ok) {
        tc_fence_after_sync();
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < CW / 32; ++c) {
          uint32_t r1_[32], r2_[32];
          tmem_ld_32x32(lane_addr + O_COL + half * CW + c * 32, r1_);
          tmem_ld_32x32(lane_addr + O_COL + DV + half * CW + c * 32, r2_);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {            // (columns past the row's width are zero)
            const float a = __uint_as_float(r1_[i]) * inv1 - __uint_as_float(r2_[i]) * inv2;
            av[c * 32 + i] = a;
            ss = fmaf(a, a, ss);
          }
        }
        float* xs = pair_max + 2 * kTcRows;         // the other buffer
        xs[half * kTcRows + row] = ss;
        __syncwarp();
        if (lane == 0) mbar_arrive(&pair_bar[q4]);
        ok = mbar_wait(&pair_bar[q4], static_cast<uint32_t>(n_tiles + 1) & 1u, p.status, kErrAttnSoftmax);
        const float rs = p.gain / sqrtf((xs[row] + xs[kTcRows + row]) / dv + p.eps);
        if (ok && row < rows_valid) {
          __nv_bfloat16* dst = p.out + static_cast<size_t>(q0 + tok0 + row) * p.out_stride + hq * dv + half * CW;
#pragma unroll
          for (int i = 0; i < CW; i += 8) {
            if (half * CW + i < dv)
              *reinterpret_cast<uint4*>(dst + i) = make_uint4(pack_bf16(av[i] * rs, av[i + 1] * rs), pack_bf16(av[i + 2] * rs, av[i + 3] * rs),
                                                              pack_bf16(av[i + 4] * rs, av[i + 5] * rs), pack_bf16(av[i + 6] * rs, av[i + 7] * rs));
          }
        }
      }
    } else {
    if constexpr (HALVES == 2) {
      if (ok && n_tiles > 0) {
        pair_sum[half * kTcRows + row] = l;
        __syncwarp();
        if (lane == 0) mbar_arrive(&pair_bar[q4]);
        ok = mbar_wait(&pair_bar[q4], static_cast<uint32_t>(n_tiles) & 1u, p.status, kErrAttnSoftmax);
        l = pair_sum[row] + pair_sum[kTcRows + row];       // (the same order in both warps)
      }
    }
    if (ok && n_tiles > 0) {
      ok = mbar_wait(pv_done, static_cast<uint32_t>(n_tiles - 1) & 1u, p.status, kErrAttnSoftmax);
    }
    if (ok) {
      tc_fence_after_sync();
      float osc = 1.0f;
      if (p.sinks != nullptr) {
        const float sk = p.sinks[hq] * 1.4426950408889634f;
        const float m2 = fmaxf(m_used, sk);
        osc = (m_used > -INFINITY) ? exp2f(m_used - m2) : 0.f;
        l = l * osc + exp2f(sk - m2);
      }
      const float inv = l > 0.f ? (EXT ? osc * p.gain : osc) / l : 0.f;
      __nv_bfloat16* dst = p.out + static_cast<size_t>(q0 + tok0 + row) * p.out_stride + hq * dv;
#pragma unroll
      for (int cc = 0; cc < DV / 32 / HALVES; ++cc) {
        const int c = half * (DV / 32 / HALVES) + cc;
        uint32_t r[32];
        tmem_ld_32x32(lane_addr + O_COL + c * 32, r);
        uint4 gv[4] = {};
        if constexpr (EXT) {
          if (gate != nullptr) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
              if (c * 32 + i * 8 < dv) gv[i] = *reinterpret_cast<const uint4*>(gate + c * 32 + i * 8);
          }
        }
        tmem_ld_wait();
        if (row < rows_valid) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if constexpr (EXT) {
              if (c * 32 + i >= dv) break;
              if (gate != nullptr) {
                const uint32_t gw[4] = {gv[i / 8].x, gv[i / 8].y, gv[i / 8].z, gv[i / 8].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                  r[i + 2 * e] = __float_as_uint(__fdividef(__uint_as_float(r[i + 2 * e]), 1.f + __expf(-bf16_lo(gw[e]))));
                  r[i + 2 * e + 1] = __float_as_uint(__fdividef(__uint_as_float(r[i + 2 * e + 1]), 1.f + __expf(-bf16_hi(gw[e]))));
                }
              }
            }
            uint4 pk;
            pk.x = pack_bf16(__uint_as_float(r[i]) * inv, __uint_as_float(r[i + 1]) * inv);
            pk.y = pack_bf16(__uint_as_float(r[i + 2]) * inv, __uint_as_float(r[i + 3]) * inv);
            pk.z = pack_bf16(__uint_as_float(r[i + 4]) * inv, __uint_as_float(r[i + 5]) * inv);
            pk.w = pack_bf16(__uint_as_float(r[i + 6]) * inv, __uint_as_float(r[i + 7]) * inv);
            *reinterpret_cast<uint4*>(dst + c * 32 + i) = pk;
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
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

template <int DK, int DV, bool EXT, int MAPS = 1, bool MEANS = false>
static int launch_prefill_tc(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const CUtensorMap& mkr, const CUtensorMap& mvm,
                             const TcPrefillParams& p, int grid, cudaStream_t stream) {
  constexpr int SUB = 128 * 128;
  constexpr int smem = (DK / 64) * SUB * (MAPS + tc_k_stages(DK, MAPS)) + (DV / 64) * SUB * tc_v_stages(DK, DV, EXT) +
                       (EXT ? 4 : 2) * SUB + 1024 + 256 + (EXT ? kExtSmem : 0);
  static_assert(smem <= 227 * 1024, "shared memory");
  auto kern = paged_prefill_tc_kernel<DK, DV, EXT, MAPS, MEANS>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    prefer_max_shared(kern);
    configured = true;
  }
  return static_cast<int>(launch_kernel(kern, dim3(grid), dim3(tc_threads(EXT)), smem, stream, mq, mk, mv, mkr, mvm, p));
}

}  // namespace mx

using namespace mx;

// Tensor-core chunked prefill over a bf16 paged pool with 16-token blocks, D = 64 or 128.
// Returns -10 when the configuration is not covered (the caller then uses mx_paged_prefill).
// `q` rows are `q_stride` elements apart (16-byte aligned, q_stride % 8 == 0); `pool_blocks` is
// the number of blocks in k_pool / v_pool; `status` is the device status word.
extern "C" int mx_paged_prefill_tc(const void* q, long long q_stride, const void* k_pool, const void* v_pool,
                                   long long pool_blocks, const int* block_tables, const int* cu_q,
                                   const int* context_lens, const float* sinks, void* out, int num_seqs,
                                   int total_q, int max_q_len, int Hq, int Hkv, int D, int block_size,
                                   int max_blocks, int window, float scale, void* status, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (num_seqs <= 0 || total_q <= 0) return 0;
  if (block_size != kTcBlock || (D != 64 && D != 128) || Hq % Hkv) return -10;
  if ((q_stride % 8) || (reinterpret_cast<uintptr_t>(q) & 15) || (reinterpret_cast<uintptr_t>(out) & 15))
    return -10;
  TcPrefillParams p{};
  p.block_tables = block_tables;
  p.cu_q = cu_q;
  p.context_lens = context_lens;
  p.sinks = sinks;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.status = static_cast<int*>(status);
  p.num_seqs = num_seqs;
  p.Hq = Hq;
  p.Hkv = Hkv;
  p.max_blocks = max_blocks;
  p.window = window;
  p.out_stride = static_cast<long long>(Hq) * D;
  p.tiles_per_seq = (max_q_len + kTcRows - 1) / kTcRows;
  p.scale_log2 = scale * 1.4426950408889634f;
  const long long grid = static_cast<long long>(num_seqs) * Hq * p.tiles_per_seq;
  if (grid > 0x7fffffffll) return -1;
  CUtensorMap mq, mk, mv;
  // q: [total_q rows, Hq * D] with row stride q_stride; box = 128 rows x 64 columns
  if (!make_tensor_map_bf16(&mq, q, static_cast<uint64_t>(total_q), static_cast<uint64_t>(Hq) * D,
                            static_cast<uint64_t>(q_stride), kTcRows, 64))
    return -4;
  // pools: [blocks * Hkv * 16 rows, D]; box = one block slab (16 rows) x 64 columns
  const uint64_t pool_rows = static_cast<uint64_t>(pool_blocks) * Hkv * kTcBlock;
  if (!make_tensor_map_bf16(&mk, k_pool, pool_rows, D, D, kTcBlock, 64)) return -4;
  if (!make_tensor_map_bf16(&mv, v_pool, pool_rows, D, D, kTcBlock, 64)) return -4;
  if (D == 64) return launch_prefill_tc<64, 64, false>(mq, mk, mv, mv, mv, p, static_cast<int>(grid), stream);
  return launch_prefill_tc<128, 128, false>(mq, mk, mv, mv, mv, p, static_cast<int>(grid), stream);
}

// Extended form: key / value rows of Dk / Dv elements (multiples of 8, at most 128); distance bias, output gate,
// chunked visibility and soft cap optional (NULL / 0). maps == 2: differential heads, Dk columns hold both maps, else gain multiplies
// the result. Output rows are out_stride elements apart. mean_rows > 0 (with a window; one map, no chunks, no bias): block means,
// k_means [mean_rows, Hkv, Dk] and v_means [mean_rows, Hkv, Dv] of blocks of mean_of tokens, sequence s from row mean_starts[s] on
// (as many as its last query sees). Returns -10 when not covered (use mx_paged_attention_any).
extern "C" int mx_paged_prefill_ext(const void* q, long long q_stride, const void* k_pool, const void* v_pool,
                                    long long pool_blocks, const int* block_tables, const int* cu_q,
                                    const int* context_lens, const float* sinks, const float* bias_r1,
                                    const float* bias_r2, const void* gate, long long gate_stride, void* out,
                                    long long out_stride, int num_seqs, int total_q, int max_q_len, int Hq, int Hkv, int Dk, int Dv,
                                    int block_size, int max_blocks, int window, int chunk, float scale, float softcap,
                                    int maps, float lambda, float gain, float eps, const void* k_means, const void* v_means,
                                    const int* mean_starts, int mean_rows, int mean_of, void* status, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (num_seqs <= 0 || total_q <= 0) return 0;
  if (Hkv <= 0 || Hq % Hkv || (bias_r1 == nullptr) != (bias_r2 == nullptr)) return -1;
  if ((maps != 1 && maps != 2) || (maps == 2 && (sinks != nullptr || bias_r1 != nullptr || gate != nullptr))) return -1;
  if (mean_rows > 0 && (window <= 0 || chunk > 0 || maps != 1 || bias_r1 != nullptr || mean_of < 1 || k_means == nullptr || v_means == nullptr ||
                        mean_starts == nullptr))
    return -1;
  const auto al16 = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) == 0; };
  if (Dk % maps) return -10;
  Dk /= maps;                          // columns of one map
  if (block_size != kTcBlock || Dk % 8 || Dv % 8 || Dk > 128 || Dv > 128 || q_stride % 8 || gate_stride % 8 || out_stride % 8 || !al16(q) ||
      !al16(out) || !al16(k_means) || !al16(v_means) || !al16(gate) || !al16(k_pool) || !al16(v_pool))
    return -10;
  TcPrefillParams p{};
  p.block_tables = block_tables;
  p.cu_q = cu_q;
  p.context_lens = context_lens;
  p.sinks = sinks;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.status = static_cast<int*>(status);
  p.num_seqs = num_seqs;
  p.Hq = Hq;
  p.Hkv = Hkv;
  p.max_blocks = max_blocks;
  p.window = window;
  p.out_stride = out_stride;
  p.gain = gain;
  p.tiles_per_seq = (max_q_len + kTcRows - 1) / kTcRows;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.dk = Dk;
  p.dv = Dv;
  p.chunk = chunk;
  p.softcap = softcap;
  p.bias_r1 = bias_r1;
  p.bias_r2 = bias_r2;
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.gate_stride = gate_stride;
  const long long grid = static_cast<long long>(num_seqs) * Hq * p.tiles_per_seq;
  if (grid > 0x7fffffffll) return -1;
  CUtensorMap mq, mk, mv;
  if (maps == 2) {
    // maps as groups of their own: a box that is wider than a map ends in zeros
    p.lambda = lambda, p.eps = eps;
    const uint64_t rows = static_cast<uint64_t>(pool_blocks) * Hkv * kTcBlock;
    if (!make_tensor_map_bf16_3d(&mq, q, total_q, 2ull * Hq, Dk, q_stride, Dk, kTcRows, 64) ||
        !make_tensor_map_bf16_3d(&mk, k_pool, rows, 2, Dk, 2ull * Dk, Dk, kTcBlock, 64) ||
        !make_tensor_map_bf16(&mv, v_pool, rows, Dv, Dv, kTcBlock, 64))
      return -4;
    const int g2 = static_cast<int>(grid);
    if (Dk <= 64)
      return Dv <= 64 ? launch_prefill_tc<64, 64, true, 2>(mq, mk, mv, mv, mv, p, g2, stream)
                      : launch_prefill_tc<64, 128, true, 2>(mq, mk, mv, mv, mv, p, g2, stream);
    return Dv <= 64 ? launch_prefill_tc<128, 64, true, 2>(mq, mk, mv, mv, mv, p, g2, stream)
                    : launch_prefill_tc<128, 128, true, 2>(mq, mk, mv, mv, mv, p, g2, stream);
  }
  // a query box may run into the next head's columns: the keys' columns there are zero
  if (!make_tensor_map_bf16(&mq, q, static_cast<uint64_t>(total_q), static_cast<uint64_t>(Hq) * Dk,
                            static_cast<uint64_t>(q_stride), kTcRows, 64))
    return -4;
  const uint64_t pool_rows = static_cast<uint64_t>(pool_blocks) * Hkv * kTcBlock;
  if (!make_tensor_map_bf16(&mk, k_pool, pool_rows, Dk, Dk, kTcBlock, 64)) return -4;
  if (!make_tensor_map_bf16(&mv, v_pool, pool_rows, Dv, Dv, kTcBlock, 64)) return -4;
  const int g = static_cast<int>(grid);
  if (mean_rows > 0) {
    p.mean_starts = mean_starts;
    p.mean_of = mean_of;
    CUtensorMap mkm, mvm;
    const uint64_t rows = static_cast<uint64_t>(mean_rows);
    if (!make_tensor_map_bf16_3d(&mkm, k_means, rows, Hkv, Dk, static_cast<uint64_t>(Hkv) * Dk, Dk, kTcKeys, 64) ||
        !make_tensor_map_bf16_3d(&mvm, v_means, rows, Hkv, Dv, static_cast<uint64_t>(Hkv) * Dv, Dv, kTcKeys, 64))
      return -4;
    if (Dk <= 64)
      return Dv <= 64 ? launch_prefill_tc<64, 64, true, 1, true>(mq, mk, mv, mkm, mvm, p, g, stream)
                      : launch_prefill_tc<64, 128, true, 1, true>(mq, mk, mv, mkm, mvm, p, g, stream);
    return Dv <= 64 ? launch_prefill_tc<128, 64, true, 1, true>(mq, mk, mv, mkm, mvm, p, g, stream)
                    : launch_prefill_tc<128, 128, true, 1, true>(mq, mk, mv, mkm, mvm, p, g, stream);
  }
  if (Dk <= 64)
    return Dv <= 64 ? launch_prefill_tc<64, 64, true>(mq, mk, mv, mv, mv, p, g, stream)
                    : launch_prefill_tc<64, 128, true>(mq, mk, mv, mv, mv, p, g, stream);
  return Dv <= 64 ? launch_prefill_tc<128, 64, true>(mq, mk, mv, mv, mv, p, g, stream)
                  : launch_prefill_tc<128, 128, true>(mq, mk, mv, mv, mv, p, g, stream);
}

// Latent attention over expanded rows: keys [k_nope (Dn) | shared rotated part (R)], values Dv wide. Sequence s owns query
// rows [cu_q[s], cu_q[s + 1]) of q (rows of heads of Dn + R elements), the last of its context_lens[s] tokens; its
// context lies in rows kv_starts[s] .. (the first of them, that of token 0, may be before the matrices where the window is not) of kn [kv_rows, H * Dn], kr (rows kr_stride apart, R used) and v [kv_rows, H * Dv].
// Output rows are out_stride elements apart. -10 = not covered.
extern "C" int mx_latent_prefill(const void* q, long long q_stride, const void* kn, const void* kr, long long kr_stride,
                                 const void* v, long long kv_rows, const int* cu_q, const int* context_lens,
                                 const int* kv_starts, const float* sinks, void* out, long long out_stride, int num_seqs,
                                 int total_q, int max_q_len, int H, int Dn, int R, int Dv, int window, float scale, void* status,
                                 void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (num_seqs <= 0 || total_q <= 0) return 0;
  if (H <= 0 || kv_rows <= 0) return -1;
  const auto al16 = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) == 0; };
  if (Dn % 8 || R % 8 || Dv % 8 || Dn <= 0 || Dn > 128 || R <= 0 || R > 64 || Dv <= 0 || Dv > 128 || q_stride % 8 || kr_stride % 8 ||
      out_stride % 8 || !al16(q) || !al16(kn) || !al16(kr) || !al16(v) || !al16(out))
    return -10;
  TcPrefillParams p{};
  p.cu_q = cu_q;
  p.context_lens = context_lens;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.status = static_cast<int*>(status);
  p.num_seqs = num_seqs;
  p.Hq = p.Hkv = H;
  p.tiles_per_seq = (max_q_len + kTcRows - 1) / kTcRows;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.dk = Dn + R;
  p.dv = Dv;
  p.kv_starts = kv_starts;
  p.sinks = sinks;
  p.gain = 1.f;
  p.window = window;
  p.kv_split = Dn;
  p.out_stride = out_stride;
  const long long grid = static_cast<long long>(num_seqs) * H * p.tiles_per_seq;
  if (grid > 0x7fffffffll) return -1;
  // a query box of the unrotated part may run into the rotated columns: the keys' columns there are zero
  CUtensorMap mq, mk, mv, mkr;
  if (!make_tensor_map_bf16_3d(&mq, q, total_q, H, Dn + R, q_stride, Dn + R, kTcRows, 64) ||
      !make_tensor_map_bf16_3d(&mk, kn, kv_rows, H, Dn, static_cast<uint64_t>(H) * Dn, Dn, kTcKeys, 64) ||
      !make_tensor_map_bf16_3d(&mv, v, kv_rows, H, Dv, static_cast<uint64_t>(H) * Dv, Dv, kTcKeys, 64) ||
      !make_tensor_map_bf16(&mkr, kr, kv_rows, R, kr_stride, kTcKeys, 64))
    return -4;
  const int g = static_cast<int>(grid);
  if (Dn <= 64)
    return Dv <= 64 ? launch_prefill_tc<128, 64, true>(mq, mk, mv, mkr, mv, p, g, stream)
                    : launch_prefill_tc<128, 128, true>(mq, mk, mv, mkr, mv, p, g, stream);
  return Dv <= 64 ? launch_prefill_tc<192, 64, true>(mq, mk, mv, mkr, mv, p, g, stream)
                  : launch_prefill_tc<192, 128, true>(mq, mk, mv, mkr, mv, p, g, stream);
}
