// Parameters the two absorbed latent decode kernels share (latent.cu: mma.sync; latent_tc.cu: tcgen05).
#pragma once
#include "common.cuh"

namespace mx {

struct LatentDecodeParams {
  const __nv_bfloat16* q;
  long long q_stride;                     // between tokens; heads are W apart
  const __nv_bfloat16* pool;
  const int* block_tables;
  const int* context_lens;
  const float* sinks;                     // exp(sinks[h]) joins the denominator (NULL: none)
  __nv_bfloat16* out;                     // [B, H, C]
  float* scratch_o;                       // [B, head tiles, splits, head_tile, C]
  float* scratch_ml;                      // [B, head tiles, splits, head_tile, 2]: (maximum, sum)
  int H, W, C, block_size, max_blocks, num_splits;
  int head_tile, head_tiles;              // heads per CTA, tiles of them
  int window;                             // > 0: the last `window` tokens only
  float scale_log2;
};

// Tokens of a split: tiles of `keys` tokens from the one that holds the window's first token on.
struct LatentSpan {
  int begin, t0, t1;                      // first visible token, tiles [t0, t1) of this split
};
__device__ __forceinline__ LatentSpan latent_span(const LatentDecodeParams& p, int len, int split, int keys) {
  const int begin = p.window > 0 ? max(0, len - p.window) : 0, first = begin / keys;
  const int tiles = (len + keys - 1) / keys, per = (tiles - first + p.num_splits - 1) / p.num_splits;
  const int t0 = first + split * per;
  return {begin, t0, min(tiles, t0 + per)};
}

// Denominator of a head whose weights sum to l relative to the maximum m (log2 units), with its sink; `scale` is what the
// value sum has to be multiplied by.
__device__ __forceinline__ float latent_denominator(const LatentDecodeParams& p, int h, float m, float l, float& scale) {
  scale = 1.f;
  if (p.sinks == nullptr) return l;
  const float sk = p.sinks[h] * 1.4426950408889634f, top = fmaxf(m, sk);
  scale = m > -INFINITY ? exp2f(m - top) : 0.f;
  return l * scale + exp2f(sk - top);
}

// The tcgen05 form (pool of pool_rows rows, 16-token blocks). -10 = not covered.
int latent_decode_tc(const LatentDecodeParams& d, int B, long long pool_rows, int* status, cudaStream_t st);

}  // namespace mx
