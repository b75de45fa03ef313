// Block means beside a paged KV pool: the mean key and value of every full run of P tokens, counted from the sequence's start.
// The mean of block b lies in the page of the block's last token, at place b - page * block_size / P (integer division) of the
// page's ceil(block_size / P) places.
//   kv_append_means   k and v rows as projected into the paged pool, and the means of the blocks these tokens complete
//   gather_means      the first means of every sequence as dense rows (the prefill kernel loads them as tiles)
#include "api.h"
#include "typed.cuh"

namespace mx {

struct MeansParams {
  const void* src;            // rows q | k | v | .., ld elements apart; k starts at column k0
  long long ld;
  const int* positions;
  const int* slots;
  const int* tables;
  const int* cu;              // row bounds of the sequences; NULL: one row each
  void *k, *v, *k_mean, *v_mean;
  int n, num_seqs, k0, Hkv, Dk, Dv, block_size, max_blocks, P, places;
};

// V consecutive elements as they lie in memory (V = 1, or 16 bytes).
template <typename T, int V>
struct Group {
  alignas(V * sizeof(T)) T v[V];
  __device__ __forceinline__ void load(const T* p) {
    if constexpr (V == 1) v[0] = *p;
    else *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(p);
  }
  __device__ __forceinline__ void store(T* p) const {
    if constexpr (V == 1) *p = v[0];
    else *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(v);
  }
};

// One thread per V elements of a token's key and value heads. A token that ends a block also sums the block up: rows of this
// call from the source (they are being appended now), earlier ones from the pool, oldest first.
template <typename T, int V>
__global__ void __launch_bounds__(256) kv_append_means_kernel(const MeansParams p) {
  constexpr int B = 4;                                    // rows of a block requested at a time
  pdl_trigger();
  pdl_wait();
  const int kg = p.Hkv * (p.Dk / V), per = kg + p.Hkv * (p.Dv / V);
  const unsigned i = blockIdx.x * 256u + threadIdx.x, tt = i / per;
  if (tt >= static_cast<unsigned>(p.n)) return;
  const int t = static_cast<int>(tt), g = static_cast<int>(i - tt * per), slot = p.slots[t], pos = p.positions[t];
  if (slot < 0) return;
  const bool key = g < kg;
  const int D = key ? p.Dk : p.Dv, j = key ? g : g - kg, head = j / (D / V), col = (j - head * (D / V)) * V;
  const T* src = static_cast<const T*>(p.src) + p.k0 + (key ? 0 : p.Hkv * p.Dk) + head * D + col;
  T* pool = static_cast<T*>(key ? p.k : p.v);
  const int blk = slot / p.block_size, off = slot - blk * p.block_size;
  Group<T, V> own;
  own.load(src + static_cast<size_t>(t) * p.ld);
  own.store(pool + ((static_cast<size_t>(blk) * p.Hkv + head) * p.block_size + off) * D + col);
  if ((pos + 1) % p.P != 0) return;
  int lo = 0, first = t;                                  // the token's sequence and its first row
  if (p.cu == nullptr) {
    lo = t;
  } else {
    int hi = p.num_seqs;
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (p.cu[mid] <= t) lo = mid;
      else hi = mid;
    }
    first = p.cu[lo];
  }
  const int* table = p.tables + static_cast<size_t>(lo) * p.max_blocks;
  float sum[V];
#pragma unroll
  for (int e = 0; e < V; ++e) sum[e] = 0.f;
  for (int back = p.P - 1; back > 0; back -= B) {
    Group<T, V> a[B];
#pragma unroll
    for (int b = 0; b < B; ++b) {
      const int k = max(back - b, 1);
      if (t - k >= first) {
        a[b].load(src + static_cast<size_t>(t - k) * p.ld);
      } else {
        const int q = pos - k, page = q / p.block_size;
        a[b].load(pool + ((static_cast<size_t>(table[page]) * p.Hkv + head) * p.block_size + (q - page * p.block_size)) * D + col);
      }
    }
#pragma unroll
    for (int b = 0; b < B; ++b)
      if (back - b > 0) {
#pragma unroll
        for (int e = 0; e < V; ++e) sum[e] += to_f(a[b].v[e]);
      }
  }
  Group<T, V> mean;
#pragma unroll
  for (int e = 0; e < V; ++e) mean.v[e] = from_f<T>((sum[e] + to_f(own.v[e])) / static_cast<float>(p.P));
  const int page = pos / p.block_size, at = (pos + 1) / p.P - 1 - page * p.block_size / p.P;
  mean.store(static_cast<T*>(key ? p.k_mean : p.v_mean) + ((static_cast<size_t>(table[page]) * p.Hkv + head) * p.places + at) * D + col);
}

// Row r of the result is block r - bounds[s] of sequence s (bounds[s] <= r < bounds[s + 1]); BYTES of it per thread.
template <int BYTES>
__global__ void __launch_bounds__(256)
gather_means_kernel(const uint8_t* __restrict__ k_mean, const uint8_t* __restrict__ v_mean, const int* __restrict__ tables,
                    const int* __restrict__ bounds, uint8_t* __restrict__ k, uint8_t* __restrict__ v, int rows, int num_seqs, int H, int kb,
                    int vb, int places, int block_size, int max_blocks, int P) {
  pdl_trigger();
  pdl_wait();
  const int kg = H * (kb / BYTES), per = kg + H * (vb / BYTES);
  const unsigned i = blockIdx.x * 256u + threadIdx.x, r = i / per;
  if (r >= static_cast<unsigned>(rows)) return;
  const int g = static_cast<int>(i - r * per);
  int lo = 0, hi = num_seqs;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (bounds[mid] <= static_cast<int>(r)) lo = mid;
    else hi = mid;
  }
  const bool key = g < kg;
  const int bytes = key ? kb : vb, j = key ? g : g - kg, head = j / (bytes / BYTES), at = (j - head * (bytes / BYTES)) * BYTES;
  const int b = static_cast<int>(r) - bounds[lo], page = ((b + 1) * P - 1) / block_size;
  const size_t row = (static_cast<size_t>(tables[static_cast<size_t>(lo) * max_blocks + page]) * H + head) * places + (b - page * block_size / P);
  const uint8_t* s = (key ? k_mean : v_mean) + row * bytes + at;
  uint8_t* d = (key ? k : v) + (static_cast<size_t>(r) * H + head) * bytes + at;
  if constexpr (BYTES == 16) *reinterpret_cast<uint4*>(d) = *reinterpret_cast<const uint4*>(s);
  else *reinterpret_cast<uint16_t*>(d) = *reinterpret_cast<const uint16_t*>(s);
}

}  // namespace mx

using namespace mx;

// Rows of one group of sequences. positions, slots [n]; tables [num_seqs, max_blocks]; cu NULL: row s is sequence s.
extern "C" int mx_kv_append_means(const void* src, long long ld, const void* positions, const void* slots, const void* tables, const void* cu,
                                  void* k, void* v, void* k_mean, void* v_mean, int n, int num_seqs, int Hq, int Hkv, int Dk,
                                  int Dv, int block_size, int max_blocks, int P, int fp32, void* stream) {
  if (n <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || Dk <= 0 || Dv <= 0 || block_size <= 0 || P <= 0 || num_seqs <= 0 || (cu == nullptr && num_seqs < n)) return -1;
  const MeansParams p{src, ld, static_cast<const int*>(positions), static_cast<const int*>(slots), static_cast<const int*>(tables),
                      static_cast<const int*>(cu), k, v, k_mean, v_mean, n, num_seqs, Hq * Dk, Hkv, Dk, Dv, block_size, max_blocks, P,
                      (block_size + P - 1) / P};
  const int V = fp32 ? 4 : 8;                             // elements of 16 bytes
  const bool vec = Dk % V == 0 && Dv % V == 0 && ld % V == 0 && aligned_to(src, 16) && aligned_to(k, 16) && aligned_to(v, 16) &&
                   aligned_to(k_mean, 16) && aligned_to(v_mean, 16);
  const long long threads = static_cast<long long>(n) * Hkv * (Dk + Dv) / (vec ? V : 1);
  if (threads > 0x7fffffffll) return -1;
  const dim3 grid(static_cast<unsigned>((threads + 255) / 256)), block(256);
  auto st = static_cast<cudaStream_t>(stream);
  if (fp32) return static_cast<int>(launch_kernel(vec ? kv_append_means_kernel<float, 4> : kv_append_means_kernel<float, 1>, grid, block, 0, st, p));
  return static_cast<int>(launch_kernel(vec ? kv_append_means_kernel<__nv_bfloat16, 8> : kv_append_means_kernel<__nv_bfloat16, 1>, grid, block, 0, st, p));
}

// kb / vb: bytes of a key and value row.
extern "C" int mx_gather_means(const void* k_mean, const void* v_mean, const void* tables, const void* bounds, void* k, void* v, int rows,
                               int num_seqs, int H, int kb, int vb, int places, int block_size, int max_blocks, int P, void* stream) {
  if (rows <= 0) return 0;
  if (num_seqs <= 0 || H <= 0 || kb <= 0 || vb <= 0 || kb % 2 || vb % 2 || block_size <= 0 || P <= 0 || places != (block_size + P - 1) / P) return -1;
  const bool wide = kb % 16 == 0 && vb % 16 == 0 && aligned_to(k_mean, 16) && aligned_to(v_mean, 16) && aligned_to(k, 16) && aligned_to(v, 16);
  const long long threads = static_cast<long long>(rows) * H * (kb + vb) / (wide ? 16 : 2);
  if (threads > 0x7fffffffll) return -1;
  return static_cast<int>(launch_kernel(wide ? gather_means_kernel<16> : gather_means_kernel<2>, dim3(static_cast<unsigned>((threads + 255) / 256)),
                                        dim3(256), 0, static_cast<cudaStream_t>(stream), static_cast<const uint8_t*>(k_mean),
                                        static_cast<const uint8_t*>(v_mean), static_cast<const int*>(tables), static_cast<const int*>(bounds),
                                        static_cast<uint8_t*>(k), static_cast<uint8_t*>(v), rows, num_seqs, H, kb, vb, places, block_size,
                                        max_blocks, P));
}
