// Shared by the retention kernels: retention.cu (single tokens, and portions token by token) and retention_tc.cu (portions in
// chunks on the tensor cores).
#pragma once
#include "typed.cuh"

namespace mx {

struct RetentionParams {
  const void* proj;          // rows q [H D] | k [H D] | v [H V] | gate [H V], ld elements apart
  long long ld;
  const int* positions;
  const float* inv_freq;     // [rot / 2]
  const float* decay;        // [H]
  float* memory;
  const int* slots;          // per piece; a negative slot marks a padding row (its output is zero)
  const int* cu;
  const int* reset;
  void* out;                 // rows of H V, ldo elements apart
  long long ldo;
  int H, D, V, rot, pieces;
  float norm_eps, gain;
};

// Scratch of the token-by-token kernels over N tokens (rows row0 .. row0 + N - 1), fp32, widths padded with zeros:
//   q [N, H, DP] | k [N, H, DP] | v [N, H, VP] | o [N, H, VP]
// and of the chunked form: cosines [N, rot / 2] | sines [N, rot / 2] | o [N, H, VP] where the heads are wider than a tile.
struct RetentionScratch {
  float *q, *k, *v, *o;
};
__host__ __device__ inline int ret_dp(int D) { return D <= 32 ? 32 : D <= 64 ? 64 : D <= 128 ? 128 : D <= 256 ? 256 : 512; }
__host__ __device__ inline int ret_vp(int V) { return (V + 31) / 32 * 32; }
__host__ __device__ inline RetentionScratch ret_scratch(float* s, long long N, int H, int D, int V) {
  RetentionScratch r;
  r.q = s;
  r.k = r.q + N * H * ret_dp(D);
  r.v = r.k + N * H * ret_dp(D);
  r.o = r.v + N * H * ret_vp(V);
  return r;
}

// Chunked form: bf16 rows, key heads of at most one tile, a rotation whose halves are whole 16-byte groups.
constexpr int kRetTile = 128;
inline bool ret_chunk_covered(int D, int V, int rot) { return D <= kRetTile && D % 8 == 0 && V % 8 == 0 && rot % 16 == 0; }
inline long long ret_chunk_floats(long long N, int H, int V, int rot) { return N * rot + (V > kRetTile ? N * H * ret_vp(V) : 0); }
int launch_retention_chunks(const RetentionParams& p, float* scratch, float* o_raw, int pieces, int row0, int N, int* status, cudaStream_t st);

}  // namespace mx
