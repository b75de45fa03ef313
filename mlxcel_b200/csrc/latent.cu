// Multi-head latent attention over a latent pool: one row [latent (C) | rotated key part (R)] per token and layer,
// shared by all heads (pool [blocks, 1, block_size, C + R]).
//   latent_append   projection row q_latent | latent | key part: q_latent normalised in place, the latent normalised and
//                   the key part rotated into the pool
//   latent_q_rope   rotates the last R dimensions of every query head (in place, or into the absorbed query row); dimensions
//                   are paired with those half the width on, or neighbours with each other
//   latent_gather   the pool rows of several sequences as one dense matrix (input of the key / value up-projections)
//   latent_decode   attention in the absorbed form: queries [q W_uk | q_rot] against the pool rows, the first C
//                   columns of the same rows as values; every row is read once for all heads; optional window and sinks
// Norms, angles, scores, softmax and accumulation are fp32.
#include "api.h"
#include "latent.cuh"
#include "mma_sync.cuh"
#include "typed.cuh"

namespace mx {

// ----------------------------------------------------------------------------- append
constexpr int kLaThreads = 256;

// One CTA per token, V elements per access.
template <typename T, int V>
__global__ void __launch_bounds__(kLaThreads)
latent_append_kernel(T* __restrict__ a, long long ld, const int* __restrict__ positions, const int* __restrict__ slots,
                     const float* __restrict__ inv_freq, float mscale, const float* __restrict__ qw,
                     const float* __restrict__ cw, T* __restrict__ pool, int Q, int C, int R, float eps, int adjacent) {
  __shared__ float red[2 * 33];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  T* row = a + static_cast<size_t>(t) * ld;
  const int slot = slots[t];
  const float pos = static_cast<float>(positions[t]);
  float s[2] = {0.f, 0.f};
#pragma unroll 4
  for (int i = threadIdx.x * V; i < Q + C; i += kLaThreads * V) {
    float f[V];
    load_v<V>(row + i, f);
#pragma unroll
    for (int e = 0; e < V; ++e) s[i < Q ? 0 : 1] += f[e] * f[e];
  }
  block_sums<2>(s, red);
  const float rq = 1.f / sqrtf(s[0] / max(Q, 1) + eps), rc = 1.f / sqrtf(s[1] / C + eps);
  T* dst = pool + static_cast<size_t>(max(slot, 0)) * (C + R);
#pragma unroll 4
  for (int i = threadIdx.x * V; i < Q + C; i += kLaThreads * V) {
    const bool query = i < Q;
    if (!query && slot < 0) break;
    float f[V], w[V];
    load_v<V>(row + i, f);
    load_v<V>(query ? qw + i : cw + (i - Q), w);
#pragma unroll
    for (int e = 0; e < V; ++e) f[e] *= (query ? rq : rc) * w[e];
    store_v<V>(query ? row + i : dst + (i - Q), f);
  }
  if (slot < 0) return;
  const int half = R / 2;
  for (int i = kLaThreads - 1 - threadIdx.x; i < half; i += kLaThreads) {      // (the last threads: they have the fewest columns)
    float sn, cs;
    sincosf(pos * inv_freq[i], &sn, &cs);
    cs *= mscale, sn *= mscale;
    const int iu = C + (adjacent ? 2 * i : i), iv = C + (adjacent ? 2 * i + 1 : half + i);
    const float u = to_f(row[Q + iu]), v = to_f(row[Q + iv]);
    dst[iu] = from_f<T>(u * cs - v * sn);
    dst[iv] = from_f<T>(v * cs + u * sn);
  }
}

// One CTA per token: its cosines and sines go to shared memory once, then the pairs of all heads.
template <typename T>
__global__ void __launch_bounds__(kLaThreads)
latent_q_rope_kernel(const T* __restrict__ q, long long ldq, int q_head, T* __restrict__ dst, long long ldd, int d_head,
                     const int* __restrict__ positions, const float* __restrict__ inv_freq, float mscale, int H, int R, int adjacent) {
  extern __shared__ float lr_smem[];
  const int half = R / 2;
  float *cs = lr_smem, *sn = lr_smem + half;
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const float pos = static_cast<float>(positions[t]);
  for (int i = threadIdx.x; i < half; i += kLaThreads) {
    float s, c;
    sincosf(pos * inv_freq[i], &s, &c);
    cs[i] = c * mscale, sn[i] = s * mscale;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < H * half; i += kLaThreads) {
    const int h = i / half, j = i - h * half;
    const int iu = adjacent ? 2 * j : j, iv = adjacent ? 2 * j + 1 : half + j;
    const T* src = q + t * ldq + static_cast<size_t>(h) * q_head;
    T* out = dst + t * ldd + static_cast<size_t>(h) * d_head;
    const float u = to_f(src[iu]), v = to_f(src[iv]);
    out[iu] = from_f<T>(u * cs[j] - v * sn[j]);
    out[iv] = from_f<T>(v * cs[j] + u * sn[j]);
  }
}

// Row r of the dense matrix is token r - zero[s] of sequence s (starts[s] <= r < starts[s + 1]).
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint8_t* __restrict__ pool, const int* __restrict__ tables, const int* __restrict__ starts,
                     const int* __restrict__ zero, uint8_t* __restrict__ out, int rows, int num_seqs, int row_bytes, int unit, int block_size, int max_blocks) {
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = blockIdx.x * 8 + warp;
  if (r >= rows) return;
  int lo = 0, hi = num_seqs;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (starts[mid] <= r) lo = mid;
    else hi = mid;
  }
  const int tok = r - zero[lo];
  const int blk = tables[static_cast<size_t>(lo) * max_blocks + tok / block_size];
  const uint8_t* src = pool + (static_cast<size_t>(blk) * block_size + tok % block_size) * row_bytes;
  uint8_t* dst = out + static_cast<size_t>(r) * row_bytes;
  if (unit == 16) {
    for (int i = lane * 16; i < row_bytes; i += 512) *reinterpret_cast<uint4*>(dst + i) = *reinterpret_cast<const uint4*>(src + i);
  } else {
    for (int i = lane * 2; i < row_bytes; i += 64) *reinterpret_cast<uint16_t*>(dst + i) = *reinterpret_cast<const uint16_t*>(src + i);
  }
}

// ----------------------------------------------------------------------------- absorbed decode
// A CTA owns (sequence, tile of 16 MT heads, KV split) and walks the split in tiles of 64 tokens, double-buffered with
// cp.async. Per tile: the eight warps take 16 tokens x half of the row's columns each for the scores (the halves are
// added in shared memory), the softmax runs over 16 threads per head, and for the values each warp owns an eighth of the
// latent columns of the SAME shared tile. Weights enter the value product as two bf16 terms (rounded weight and
// remainder). Splits leave fp32 partial results for a merge kernel (one CTA per head row).
constexpr float kLdLog2e = 1.4426950408889634f;
constexpr int kLdThreads = 256, kLdKeys = 64, kLdMaxRow = 576, kLdMaxLatent = 512;
constexpr int kLdSRow = kLdKeys + 4;      // floats per score row
constexpr int kLdPRow = kLdKeys + 8;      // bf16 per weight row (an odd number of 16-byte chunks)

__host__ __device__ inline int ld_row_bytes(int W) { return (W + 15) / 16 * 32 + 16; }   // an odd number of 16-byte chunks
__host__ inline int ld_smem(int W, int mt) {
  return (16 * mt + 2 * kLdKeys) * ld_row_bytes(W) + 2 * 16 * mt * kLdSRow * 4 + 2 * 16 * mt * kLdPRow * 2;
}

template <int MT>
__global__ void __launch_bounds__(kLdThreads, 1) latent_decode_kernel(const LatentDecodeParams p) {
  constexpr int HR = 16 * MT;             // head rows of the tile
  extern __shared__ __align__(128) uint8_t ld_sm[];
  const int RS = ld_row_bytes(p.W), KS = (p.W + 15) / 16;   // row stride, 16-column steps
  uint8_t* q_s = ld_sm;
  uint8_t* k_s = q_s + HR * RS;
  float* s_s = reinterpret_cast<float*>(k_s + 2 * kLdKeys * RS);                       // [2 halves][HR][kLdSRow]
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(s_s + 2 * HR * kLdSRow);       // [2 terms][HR][kLdPRow]
  __shared__ float alpha_s[HR], m_s[HR], l_s[HR];
  pdl_trigger();

  const int split = blockIdx.x % p.num_splits, bt = blockIdx.x / p.num_splits;
  const int ht = bt % p.head_tiles, b = bt / p.head_tiles;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h0 = ht * HR, heads = min(HR, p.H - h0);
  const int len = p.context_lens[b];
  const LatentSpan span = latent_span(p, len, split, kLdKeys);
  const int t0 = span.t0, t1 = span.t1;
  const int* table = p.block_tables + static_cast<size_t>(b) * p.max_blocks;
  const int chunks = p.W / 8, row_chunks = KS * 2;          // real and padded 16-byte chunks of a row
  pdl_wait();

  for (int i = threadIdx.x; i < HR * row_chunks; i += kLdThreads) {
    const int r = i / row_chunks, c = i - r * row_chunks;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < heads && c < chunks)
      v = *reinterpret_cast<const uint4*>(p.q + static_cast<size_t>(b) * p.q_stride + static_cast<size_t>(h0 + r) * p.W + c * 8);
    *reinterpret_cast<uint4*>(q_s + r * RS + c * 16) = v;
  }
  if (threadIdx.x < HR) m_s[threadIdx.x] = -INFINITY, l_s[threadIdx.x] = 0.f;

  // four threads per token; rows past the end and columns past the row are zero-filled
  const auto load_tile = [&](int tile, int stage) {
    if (tile < t1) {
      const int r = threadIdx.x >> 2, key = tile * kLdKeys + r;
      const bool ok = key < len;
      const size_t prow = ok ? static_cast<size_t>(table[key / p.block_size]) * p.block_size + key % p.block_size : 0;
      const __nv_bfloat16* src = p.pool + prow * p.W;
      const uint32_t dst = smem_u32(k_s + (stage * kLdKeys + r) * RS);
      for (int c = threadIdx.x & 3; c < row_chunks; c += 4) {
        const bool in = ok && c < chunks;
        cp_async16(dst + c * 16, in ? src + c * 8 : p.pool, in);
      }
    }
    cp_async_commit();
  };

  const int NT = (p.C + 15) / 16;         // 16-column value tiles: warp w takes w, w + 8, ...
  float o[MT][4][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 8; ++e) o[m][n][e >> 2][e & 3] = 0.f;

  load_tile(t0, 0);
  for (int tile = t0; tile < t1; ++tile) {
    const int stage = (tile - t0) & 1;
    load_tile(tile + 1, stage ^ 1);       // (its previous reader finished before the barrier at the loop's end)
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t kb = smem_u32(k_s + stage * kLdKeys * RS);
    {
      // ---- scores: tokens kg .. + 15, columns of half kh
      const int kg = (warp & 3) * 16, kh = warp >> 2;
      const int k0 = kh == 0 ? 0 : KS / 2, k1 = kh == 0 ? KS / 2 : KS;
      float sc[MT][2][4], sd[MT][2][4];   // even and odd steps: independent accumulation chains
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int e = 0; e < 8; ++e) sc[m][e >> 2][e & 3] = sd[m][e >> 2][e & 3] = 0.f;
      const uint32_t ka = kb + (kg + (lane & 7) + (lane >> 4) * 8) * RS + ((lane >> 3) & 1) * 16;
      const uint32_t qa = smem_u32(q_s) + ((lane & 7) + ((lane >> 3) & 1) * 8) * RS + (lane >> 4) * 16;
      const auto step = [&](int kk, float(&acc)[MT][2][4]) {
        uint32_t kf[4];
        ldmatrix_x4(kf, ka + kk * 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t qf[4];
          ldmatrix_x4(qf, qa + m * 16 * RS + kk * 32);
          mma_bf16_16816(acc[m][0], qf, kf[0], kf[1]);
          mma_bf16_16816(acc[m][1], qf, kf[2], kf[3]);
        }
      };
      int kk = k0;
#pragma unroll 3
      for (; kk + 1 < k1; kk += 2) {
        step(kk, sc);
        step(kk + 1, sd);
      }
      if (kk < k1) step(kk, sc);
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int e = 0; e < 8; ++e) sc[m][e >> 2][e & 3] += sd[m][e >> 2][e & 3];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          float* d = s_s + (kh * HR + m * 16 + (lane >> 2)) * kLdSRow + kg + n * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(d) = make_float2(sc[m][n][0], sc[m][n][1]);
          *reinterpret_cast<float2*>(d + 8 * kLdSRow) = make_float2(sc[m][n][2], sc[m][n][3]);
        }
    }
    __syncthreads();
    // ---- softmax: 16 threads per head, four tokens each
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int r = m * 16 + (threadIdx.x >> 4), c = (threadIdx.x & 15) * 4;
      const float4 x = *reinterpret_cast<const float4*>(s_s + r * kLdSRow + c);
      const float4 y = *reinterpret_cast<const float4*>(s_s + (HR + r) * kLdSRow + c);
      float v[4] = {x.x + y.x, x.y + y.y, x.z + y.z, x.w + y.w};
      float mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = tile * kLdKeys + c + e;
        v[e] = key < len && key >= span.begin ? v[e] * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, v[e]);
      }
#pragma unroll
      for (int d = 8; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float m_old = m_s[r], mn = fmaxf(m_old, mx);     // (a tile below t1 has a visible token: mn is finite)
      float sum = 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[e] = exp2f(v[e] - mn);
        sum += v[e];
      }
#pragma unroll
      for (int d = 8; d > 0; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
      const uint32_t a0 = pack_bf16(v[0], v[1]), a1 = pack_bf16(v[2], v[3]);
      *reinterpret_cast<uint2*>(p_s + r * kLdPRow + c) = make_uint2(a0, a1);
      *reinterpret_cast<uint2*>(p_s + (HR + r) * kLdPRow + c) =
          make_uint2(pack_bf16(v[0] - bf16_lo(a0), v[1] - bf16_hi(a0)), pack_bf16(v[2] - bf16_lo(a1), v[3] - bf16_hi(a1)));
      __syncwarp();
      if ((threadIdx.x & 15) == 0) {
        const float al = m_old > -INFINITY ? exp2f(m_old - mn) : 0.f;
        alpha_s[r] = al;
        m_s[r] = mn;
        l_s[r] = l_s[r] * al + sum;
      }
    }
    __syncthreads();
    // ---- values
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float a_lo = alpha_s[m * 16 + (lane >> 2)], a_hi = alpha_s[m * 16 + 8 + (lane >> 2)];
      if (__any_sync(0xffffffffu, a_lo != 1.f || a_hi != 1.f)) {
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int j = 0; j < 2; ++j) o[m][n][j][0] *= a_lo, o[m][n][j][1] *= a_lo, o[m][n][j][2] *= a_hi, o[m][n][j][3] *= a_hi;
      }
    }
    const uint32_t va = kb + ((lane & 7) + ((lane >> 3) & 1) * 8) * RS + (lane >> 4) * 16;
    const uint32_t pa = smem_u32(p_s) + ((lane & 7) + ((lane >> 3) & 1) * 8) * (kLdPRow * 2) + (lane >> 4) * 16;
#pragma unroll
    for (int kk = 0; kk < kLdKeys / 16; ++kk) {
      uint32_t w[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int term = 0; term < 2; ++term) ldmatrix_x4(w[m][term], pa + ((term * HR + m * 16) * kLdPRow + kk * 16) * 2);
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int nt = warp + n * 8;
        if (nt >= NT) continue;           // (the same for the whole warp)
        uint32_t vf[4];
        ldmatrix_x4_trans(vf, va + kk * 16 * RS + nt * 32);
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int term = 0; term < 2; ++term) {
            mma_bf16_16816(o[m][n][0], w[m][term], vf[0], vf[1]);
            mma_bf16_16816(o[m][n][1], w[m][term], vf[2], vf[3]);
          }
      }
    }
    __syncthreads();                      // the tile and the weights may be overwritten
  }
  cp_async_wait<0>();
  __syncthreads();

  // ---- results of this split
  const size_t part = static_cast<size_t>(bt) * p.num_splits + split;
  float* po = p.scratch_o + part * HR * p.C;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int r = m * 16 + (lane >> 2) + ((e & 2) ? 8 : 0);
        const int c = (warp + n * 8) * 16 + (e >> 2) * 8 + (lane & 3) * 2 + (e & 1);
        if (r >= heads || c >= p.C) continue;
        const float v = o[m][n][e >> 2][e & 3];
        if (p.num_splits > 1) {
          po[r * p.C + c] = v;
        } else {
          float f;
          const float l = latent_denominator(p, h0 + r, m_s[r], l_s[r], f);
          p.out[(static_cast<size_t>(b) * p.H + h0 + r) * p.C + c] = __float2bfloat16(l > 0.f ? v * f / l : 0.f);
        }
      }
  if (p.num_splits == 1) return;
  if (threadIdx.x < HR) {
    p.scratch_ml[(part * HR + threadIdx.x) * 2] = m_s[threadIdx.x];
    p.scratch_ml[(part * HR + threadIdx.x) * 2 + 1] = l_s[threadIdx.x];
  }
}

// out[b, h, :] from the partial results of its splits; one CTA per (sequence, head), two columns per thread.
__global__ void __launch_bounds__(256) latent_merge_kernel(const LatentDecodeParams p) {
  __shared__ float f_s[64];
  __shared__ float inv_s;
  pdl_trigger();
  pdl_wait();
  const int HR = p.head_tile, b = blockIdx.x / p.H, h = blockIdx.x - b * p.H, ht = h / HR, r = h - ht * HR;
  const size_t base = (static_cast<size_t>(b) * p.head_tiles + ht) * p.num_splits;
  if (threadIdx.x < 32) {
    float m[2], l[2], mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = threadIdx.x + i * 32;
      m[i] = s < p.num_splits ? p.scratch_ml[((base + s) * HR + r) * 2] : -INFINITY;
      l[i] = s < p.num_splits ? p.scratch_ml[((base + s) * HR + r) * 2 + 1] : 0.f;
      mx = fmaxf(mx, m[i]);
    }
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const float f = m[i] > -INFINITY ? exp2f(m[i] - mx) : 0.f;
      f_s[threadIdx.x + i * 32] = f;
      sum += f * l[i];
    }
    sum = warp_sum(sum);
    if (threadIdx.x == 0) {
      float f;
      const float l = latent_denominator(p, h, mx, sum, f);
      inv_s = l > 0.f ? f / l : 0.f;
    }
  }
  __syncthreads();
  for (int c = threadIdx.x * 2; c < p.C; c += 512) {
    const float* o = p.scratch_o + (base * HR + r) * static_cast<size_t>(p.C) + c;
    float x = 0.f, y = 0.f;
#pragma unroll 8
    for (int s = 0; s < p.num_splits; ++s) {
      const float2 v = *reinterpret_cast<const float2*>(o + static_cast<size_t>(s) * HR * p.C);
      x += f_s[s] > 0.f ? f_s[s] * v.x : 0.f, y += f_s[s] > 0.f ? f_s[s] * v.y : 0.f;   // (a split without tokens wrote nothing)
    }
    *reinterpret_cast<uint32_t*>(p.out + (static_cast<size_t>(b) * p.H + h) * p.C + c) = pack_bf16(x * inv_s, y * inv_s);
  }
}

template <int MT>
static int launch_latent_decode(const LatentDecodeParams& p, int grid, cudaStream_t st) {
  auto kern = latent_decode_kernel<MT>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, ld_smem(kLdMaxRow, MT));
    if (e != cudaSuccess) return static_cast<int>(e);
    prefer_max_shared(kern);
    configured = true;
  }
  return static_cast<int>(launch_kernel(kern, dim3(grid), dim3(kLdThreads), ld_smem(p.W, MT), st, p));
}

}  // namespace mx

using namespace mx;

constexpr int kLatentScratch0 = 65536;    // the scratch buffer starts with the counters of the paged decode kernels

// a: rows q_latent [Q] | latent [C] | key part [R], ld elements apart. Q may be 0.
extern "C" int mx_latent_append(void* a, long long ld, const void* positions, const void* slots, const void* inv_freq, float mscale,
                                const void* qw, const void* cw, void* pool, int n, int Q, int C, int R, float eps, int adjacent,
                                int fp32, void* stream) {
  if (n <= 0) return 0;
  if (Q < 0 || C <= 0 || R < 0 || R % 2 || (Q > 0 && qw == nullptr)) return -1;
  auto st = static_cast<cudaStream_t>(stream);
  const size_t ab = fp32 ? 16 : 8;
  const bool vec = Q % 4 == 0 && C % 4 == 0 && R % 4 == 0 && ld % 4 == 0 && aligned_to(a, ab) && aligned_to(pool, ab) && aligned_to(qw, 16) &&
                   aligned_to(cw, 16);
#define MX_LA(T, V)                                                                                                           \
  return static_cast<int>(launch_kernel(latent_append_kernel<T, V>, dim3(n), dim3(kLaThreads), 0, st, static_cast<T*>(a), ld,    \
                                        static_cast<const int*>(positions), static_cast<const int*>(slots),                   \
                                        static_cast<const float*>(inv_freq), mscale, static_cast<const float*>(qw),           \
                                        static_cast<const float*>(cw), static_cast<T*>(pool), Q, C, R, eps, adjacent))
  if (fp32) {
    if (vec) MX_LA(float, 4);
    MX_LA(float, 1);
  }
  if (vec) MX_LA(__nv_bfloat16, 4);
  MX_LA(__nv_bfloat16, 1);
#undef MX_LA
}

// q / dst point at the first rotated dimension of the first head; heads are q_head / d_head, tokens ldq / ldd elements apart.
extern "C" int mx_latent_q_rope(const void* q, long long ldq, int q_head, void* dst, long long ldd, int d_head, const void* positions,
                                const void* inv_freq, float mscale, int n, int H, int R, int adjacent, int fp32, void* stream) {
  if (n <= 0 || R == 0) return 0;
  if (H <= 0 || R < 0 || R % 2 || R > 8192) return -1;
  auto st = static_cast<cudaStream_t>(stream);
#define MX_LQ(T)                                                                                                              \
  return static_cast<int>(launch_kernel(latent_q_rope_kernel<T>, dim3(n), dim3(kLaThreads), R * sizeof(float), st,            \
                                        static_cast<const T*>(q), ldq, q_head, static_cast<T*>(dst), ldd, d_head,             \
                                        static_cast<const int*>(positions), static_cast<const float*>(inv_freq), mscale, H, R, adjacent))
  if (fp32) MX_LQ(float);
  MX_LQ(__nv_bfloat16);
#undef MX_LQ
}

extern "C" int mx_latent_gather(const void* pool, const void* tables, const void* starts, const void* zero, void* out, int rows,
                                int num_seqs, int row_bytes, int block_size, int max_blocks, void* stream) {
  if (rows <= 0) return 0;
  if (num_seqs <= 0 || row_bytes <= 0 || row_bytes % 2 || block_size <= 0) return -1;
  const int unit = row_bytes % 16 == 0 && aligned_to(pool, 16) && aligned_to(out, 16) ? 16 : 2;
  return static_cast<int>(launch_kernel(latent_gather_kernel, dim3((rows + 7) / 8), dim3(256), 0, static_cast<cudaStream_t>(stream),
                                        static_cast<const uint8_t*>(pool), static_cast<const int*>(tables),
                                        static_cast<const int*>(starts), static_cast<const int*>(zero), static_cast<uint8_t*>(out), rows, num_seqs, row_bytes,
                                        unit, block_size, max_blocks));
}

// Heads per CTA tile and the scratch floats of a call.
extern "C" int mx_latent_head_tile(int H) { return H > 16 ? 32 : 16; }
extern "C" long long mx_latent_decode_scratch_floats(int B, int H, int C, int num_splits) {
  const int hr = mx_latent_head_tile(H);
  return kLatentScratch0 + static_cast<long long>(B) * ((H + hr - 1) / hr) * hr * num_splits * (C + 2);
}

// Absorbed queries [B, H, W] (token stride q_stride) over the latent pool (pool_rows rows) -> out [B, H, C]. form 0: the
// tcgen05 kernel where it applies (16-token blocks), else the mma.sync one; 1: the mma.sync one. bf16; W at most 576, C at most
// 512, multiples of 8. -10 = not covered (use mx_paged_attention_any).
extern "C" int mx_latent_decode(const void* q, long long q_stride, const void* pool, long long pool_rows, const void* block_tables,
                                const void* context_lens, const void* sinks, void* out, float* scratch, int B, int H, int W, int C,
                                int block_size, int max_blocks, int window, float scale, int num_splits, int form, void* status, void* stream) {
  if (B <= 0) return 0;
  if (H <= 0 || C <= 0 || C > W || block_size <= 0) return -1;
  if (W % 8 || C % 8 || W > kLdMaxRow || C > kLdMaxLatent || q_stride % 8 || !aligned_to(q, 16) || !aligned_to(pool, 16)) return -10;
  if (num_splits < 1) num_splits = 1;
  if (num_splits > 64) num_splits = 64;
  const int hr = mx_latent_head_tile(H);
  LatentDecodeParams p{};
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.q_stride = q_stride;
  p.pool = static_cast<const __nv_bfloat16*>(pool);
  p.block_tables = static_cast<const int*>(block_tables);
  p.context_lens = static_cast<const int*>(context_lens);
  p.sinks = static_cast<const float*>(sinks);
  p.window = window;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.H = H, p.W = W, p.C = C, p.block_size = block_size, p.max_blocks = max_blocks, p.num_splits = num_splits;
  p.head_tile = hr, p.head_tiles = (H + hr - 1) / hr;
  p.scale_log2 = scale * kLdLog2e;
  const long long pairs = static_cast<long long>(B) * p.head_tiles;
  if (pairs * num_splits > 0x7fffffffll || static_cast<long long>(B) * H > 0x7fffffffll) return -1;
  p.scratch_ml = scratch + kLatentScratch0;
  p.scratch_o = p.scratch_ml + pairs * num_splits * hr * 2;
  const int grid = static_cast<int>(pairs * num_splits);
  auto st = static_cast<cudaStream_t>(stream);
  int rc = form == 1 ? -10 : latent_decode_tc(p, B, pool_rows, static_cast<int*>(status), st);
  if (rc == -10) rc = hr == 32 ? launch_latent_decode<2>(p, grid, st) : launch_latent_decode<1>(p, grid, st);
  if (rc != 0 || num_splits == 1) return rc;
  return static_cast<int>(launch_kernel(latent_merge_kernel, dim3(static_cast<unsigned>(B) * H), dim3(256), 0, st, p));
}
