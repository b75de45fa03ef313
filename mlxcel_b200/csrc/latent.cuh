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
  __nv_bfloat16* out;                     // [B, H, C]
  float* scratch_o;                       // [B, head tiles, splits, head_tile, C]
  float* scratch_ml;                      // [B, head tiles, splits, head_tile, 2]: (maximum, sum)
  int H, W, C, block_size, max_blocks, num_splits;
  int head_tile, head_tiles;              // heads per CTA, tiles of them
  float scale_log2;
};

// The tcgen05 form (pool of pool_rows rows, 16-token blocks). -10 = not covered.
int latent_decode_tc(const LatentDecodeParams& d, int B, long long pool_rows, int* status, cudaStream_t st);

}  // namespace mx
