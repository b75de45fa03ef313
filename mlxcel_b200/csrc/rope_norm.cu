// Rotary positions with a norm BEHIND them, and the KV append, for bf16 and fp32 activations:
//   rope_norm_append   rows q | k (| v): the first `rot` dimensions of every query and key head are rotated (half
//                      layout: i with i + rot / 2), then the head is divided by its root mean square and
//                      multiplied by an optional weight; queries stay in place, keys go to the paged pool, values
//                      go there as they are (either v columns, or the key columns as projected)
// Angles, cosines, rotation and norm are fp32. Frequencies arrive as a table (any scaling is in it) and `mscale`
// multiplies cosine and sine.
#include "api.h"
#include "typed.cuh"

namespace mx {

constexpr int kRnWarps = 8;

// One CTA per token (several, over the heads, when there are few tokens); the token's cosines and sines are computed once into shared memory, then a warp takes every
// eighth head: it stages the head in shared memory (the partner of a dimension sits in another lane), rotates,
// sums squares and writes. `unit`: divide by the root mean square (mean over D, eps inside the root).
template <typename T, int V>
__global__ void __launch_bounds__(kRnWarps * 32)
rope_norm_append_kernel(T* __restrict__ qkv, long long ld, const int* __restrict__ positions, const int* __restrict__ slots,
                        const float* __restrict__ inv_freq, float mscale, T* __restrict__ k_pool, T* __restrict__ v_pool,
                        const float* __restrict__ qw, const float* __restrict__ kw, int Hq, int Hkv, int Dk, int Dv, int rot,
                        int values_are_keys, int unit, int block_size, float eps) {
  extern __shared__ __align__(16) float rn_smem[];
  const int half = rot / 2, half_pad = (half + 3) & ~3, dpad = (Dk + 3) & ~3;
  float* cs = rn_smem;                     // [half]
  float* sn = cs + half_pad;               // [half]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x;
  float* hs = sn + half_pad + warp * dpad; // this warp's head
  pdl_trigger();
  pdl_wait();
  const float pos = static_cast<float>(positions[t]);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(pos * inv_freq[i], &s, &c);
    cs[i] = c * mscale;
    sn[i] = s * mscale;
  }
  __syncthreads();
  T* row = qkv + static_cast<size_t>(t) * ld;
  const int slot = slots[t];
  const int blk = slot >= 0 ? slot / block_size : 0, off = slot >= 0 ? slot - blk * block_size : 0;
  const int nv = values_are_keys ? 0 : Hkv;
  for (int hd = blockIdx.y * kRnWarps + warp; hd < Hq + Hkv + nv; hd += kRnWarps * gridDim.y) {
    if (hd >= Hq && slot < 0) break;
    if (hd >= Hq + Hkv) {                  // plain value head
      const int g = hd - Hq - Hkv;
      const T* src = row + static_cast<size_t>(Hq + Hkv) * Dk + static_cast<size_t>(g) * Dv;
      T* dst = v_pool + ((static_cast<size_t>(blk) * Hkv + g) * block_size + off) * Dv;
      for (int c = lane * V; c < Dv; c += 32 * V) {
        float f[V];
        load_v<V>(src + c, f);
        store_v<V>(dst + c, f);
      }
      continue;
    }
    const bool key = hd >= Hq;
    const int g = hd - Hq;
    T* src = row + static_cast<size_t>(hd) * Dk;
    const size_t prow = key ? (static_cast<size_t>(blk) * Hkv + g) * block_size + off : 0;
    T* dst = key ? k_pool + prow * Dk : src;
    const float* w = key ? kw : qw;
    for (int c = lane * V; c < Dk; c += 32 * V) {
      float f[V];
      load_v<V>(src + c, f);
#pragma unroll
      for (int e = 0; e < V; ++e) hs[c + e] = f[e];
      if (key && values_are_keys) store_v<V>(v_pool + prow * Dk + c, f);
    }
    __syncwarp();
    for (int i = lane; i < half; i += 32) {
      const float u = hs[i], v = hs[i + half];
      hs[i] = u * cs[i] - v * sn[i];
      hs[i + half] = v * cs[i] + u * sn[i];
    }
    __syncwarp();
    float r = 1.f;
    if (unit) {
      float s = 0.f;
      for (int c = lane; c < Dk; c += 32) s += hs[c] * hs[c];
      r = 1.f / sqrtf(warp_sum(s) / Dk + eps);
    }
    for (int c = lane * V; c < Dk; c += 32 * V) {
      float o[V];
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = hs[c + e] * r * (w != nullptr ? w[c + e] : 1.f);
      store_v<V>(dst + c, o);
    }
    __syncwarp();
  }
}

}  // namespace mx

using namespace mx;

// rot: even, at most Dk (0: no rotation). values_are_keys: rows are q | k, Dv must equal Dk. unit 0 leaves the norm out
// (the weights then act alone). qw / kw may be NULL. Tokens with a negative slot append nothing.
extern "C" int mx_rope_norm_append(void* qkv, long long ld, const void* positions, const void* slots, const void* inv_freq,
                                   float mscale, void* k_pool, void* v_pool, const void* qw, const void* kw, int n, int Hq,
                                   int Hkv, int Dk, int Dv, int rot, int values_are_keys, int unit, int block_size, float eps,
                                   int fp32, void* stream) {
  if (n <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || Dk <= 0 || Dv <= 0 || block_size <= 0 || rot < 0 || rot > Dk || rot % 2 ||
      (rot > 0 && inv_freq == nullptr) || (values_are_keys && Dk != Dv))
    return -1;
  const size_t smem = (2 * static_cast<size_t>((rot / 2 + 3) & ~3) + kRnWarps * static_cast<size_t>((Dk + 3) & ~3)) * sizeof(float);
  if (smem > 48 * 1024) return -1;
  const size_t ab = fp32 ? 16 : 8;
  const bool vec = Dk % 4 == 0 && Dv % 4 == 0 && ld % 4 == 0 && aligned_to(qkv, ab) && aligned_to(k_pool, ab) && aligned_to(v_pool, ab);
  auto st = static_cast<cudaStream_t>(stream);
  const int groups = (Hq + (values_are_keys ? 1 : 2) * Hkv + kRnWarps - 1) / kRnWarps;
  const dim3 grid(n, n >= 512 ? 1 : groups), block(kRnWarps * 32);
#define MX_RN(T, V)                                                                                                         \
  return static_cast<int>(launch_kernel(rope_norm_append_kernel<T, V>, grid, block, smem, st, static_cast<T*>(qkv), ld,     \
                                        static_cast<const int*>(positions), static_cast<const int*>(slots),                 \
                                        static_cast<const float*>(inv_freq), mscale, static_cast<T*>(k_pool),               \
                                        static_cast<T*>(v_pool), static_cast<const float*>(qw), static_cast<const float*>(kw), \
                                        Hq, Hkv, Dk, Dv, rot, values_are_keys, unit, block_size, eps))
  if (fp32) {
    if (vec) MX_RN(float, 4);
    MX_RN(float, 1);
  }
  if (vec) MX_RN(__nv_bfloat16, 4);
  MX_RN(__nv_bfloat16, 1);
#undef MX_RN
}
