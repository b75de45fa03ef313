// Shape-agnostic SIMT kernels with fp32 arithmetic, for fp32 models and for sizes the tensor-core
// kernels do not cover (row strides that are not a multiple of 16 bytes, head widths other than
// multiples of 8 up to 128):
//   gemm_any       out[M, N] = x[M, K] w[N, K]^T (+ bias) (+ residual), operands bf16 or fp32; optionally a batch of such
//                  products at constant strides (block-diagonal weights)
//   grouped_gemm_any  rows offsets[e] .. of a permuted row list times expert e's matrix
//   attention_any  causal paged attention of any query rows (decode rows are pieces of one token):
//                  sliding window, chunks, soft cap, sinks, logarithmic distance bias, output gate, key and value heads
//                  of different width (which may lie in rows wider than they are), differential heads of two maps, block means
#include "api.h"
#include "typed.cuh"

namespace mx {

// ----------------------------------------------------------------------------- GEMM
constexpr int kGaTile = 64, kGaK = 16, kGaThreads = 256;

// One tile of out[rows, N] = x[rows, K] w[N, K]^T from row m0 on; row m of x is row_map[m] where there is a map.
template <typename T, typename TO>
__device__ __forceinline__ void gemm_any_tile(const T* __restrict__ x, const T* __restrict__ w, TO* __restrict__ out,
                                              const T* __restrict__ bias, const T* __restrict__ residual,
                                              const int* __restrict__ row_map, int m0, int n0, int M, int N, int K, long long ldx,
                                              long long ldw, long long ldo, long long ldr) {
  __shared__ __align__(16) float xs[kGaK][kGaTile + 4];
  __shared__ __align__(16) float ws[kGaK][kGaTile + 4];
  const int tm = (threadIdx.x / 16) * 4, tn = (threadIdx.x % 16) * 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += kGaK) {
    __syncthreads();
    for (int i = threadIdx.x; i < kGaTile * kGaK; i += kGaThreads) {
      const int r = i / kGaK, k = i - r * kGaK;
      const bool kin = k0 + k < K, min = m0 + r < M;
      const int xr = min && row_map != nullptr ? row_map[m0 + r] : m0 + r;
      xs[k][r] = (kin && min) ? to_f(x[static_cast<size_t>(xr) * ldx + k0 + k]) : 0.f;
      ws[k][r] = (kin && n0 + r < N) ? to_f(w[static_cast<size_t>(n0 + r) * ldw + k0 + k]) : 0.f;
    }
    __syncthreads();
    // each K slice is summed on its own first: the rounding error grows with K / 16, not with K
    float part[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) part[i][j] = 0.f;
#pragma unroll
    for (int k = 0; k < kGaK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][tm]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[k][tn]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) part[i][j] = fmaf(av[i], bv[j], part[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j];
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + tm + i;
    if (m >= M) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tn + j;
      if (n >= N) break;
      float v = acc[i][j];
      if (bias != nullptr) v += to_f(bias[n]);
      if (residual != nullptr) v += to_f(residual[static_cast<size_t>(m) * ldr + n]);
      out[static_cast<size_t>(m) * ldo + n] = from_f<TO>(v);
    }
  }
}

template <typename T, typename TO>
__global__ void __launch_bounds__(kGaThreads)
gemm_any_kernel(const T* __restrict__ x, const T* __restrict__ w, TO* __restrict__ out, const T* __restrict__ bias,
                const T* __restrict__ residual, int M, int N, int K, long long ldx, long long ldw, long long ldo,
                long long ldr, long long bx, long long bw, long long bo) {
  pdl_trigger();
  pdl_wait();
  gemm_any_tile<T, TO>(x + blockIdx.z * bx, w + blockIdx.z * bw, out + blockIdx.z * bo, bias, residual, nullptr, blockIdx.y * kGaTile,
                       blockIdx.x * kGaTile, M, N, K, ldx, ldw, ldo, ldr);
}

// Rows offsets[e] .. offsets[e + 1] - 1 of the list (row r of x is row_map[r], or r itself) times w[e].
template <typename T>
__global__ void __launch_bounds__(kGaThreads)
grouped_gemm_any_kernel(const T* __restrict__ x, const T* __restrict__ w, T* __restrict__ out, const int* __restrict__ offsets,
                        const int* __restrict__ row_map, int N, int K, long long ldx) {
  pdl_trigger();
  pdl_wait();
  const int e = blockIdx.z, m0 = offsets[e] + blockIdx.y * kGaTile, m1 = offsets[e + 1];
  if (m0 >= m1) return;
  gemm_any_tile<T, T>(x, w + static_cast<size_t>(e) * N * K, out, nullptr, nullptr, row_map, m0, blockIdx.x * kGaTile, m1, N, K, ldx, K, N, 0);
}

// ----------------------------------------------------------------------------- attention
constexpr int kAaWarps = 4;

struct AnyAttnParams {
  const void* q;
  long long q_stride;
  const void* k_pool;
  const void* v_pool;
  const int* block_tables;
  const int* cu_q;
  const int* context_lens;
  const float* sinks;
  const float* r1;         // distance bias: r1[h] ln(1 + r2[h] (i - j)) is taken off the score
  const float* r2;
  const void* gate;        // the output is multiplied by sigmoid(gate)
  long long gate_stride;
  void* out;
  int num_seqs, Hq, Hkv, Dk, Dv, ldk, ldv, block_size, max_blocks, window, chunk;   // ldk / ldv: elements of a pool row
  float scale, softcap;
  // maps == 2: differential heads. Query and key rows of a head hold two maps of Dk columns each (attentions of their own
  // over the same values); the result is (a1 - lambda a2) / rms(.) * gain.
  // With one map, gain is a plain factor of the result.
  int maps;
  float lambda, gain, eps;
  long long out_stride;
  // mean_of > 0 (with a window): the mean key and value of every block of mean_of tokens wholly before the window are keys too;
  // that of block b is at place b - page * block_size / mean_of of the page that holds the block's last token.
  const void* k_mean;
  const void* v_mean;
  int mean_of, mean_rows;
};

// One CTA per (query row, query head). The warps take the 32-key chunks in turn: scores with one key
// per lane, then values with the head's dims over the lanes (NV accumulators each); each warp keeps its
// own running maximum and sum, merged at the end.
template <typename T, int NV>
__global__ void __launch_bounds__(kAaWarps * 32)
attention_any_kernel(const AnyAttnParams p) {
  extern __shared__ float aa_smem[];
  float* q_s = aa_smem;                                  // [Dk]
  float* o_s = q_s + p.Dk;                               // [warps][Dv]
  float* a_s = o_s + kAaWarps * p.Dv;                    // maps == 2: the first map's result [Dv]
  __shared__ float m_s[kAaWarps], l_s[kAaWarps], red[33];
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x, h = blockIdx.y, hk = h / (p.Hq / p.Hkv);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int lo = 0, hi = p.num_seqs;                           // sequence s with cu[s] <= row < cu[s + 1]
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (p.cu_q[mid] <= row) lo = mid;
    else hi = mid;
  }
  const int s = lo;
  if (row < p.cu_q[s] || row >= p.cu_q[s + 1]) return;
  const int pos = p.context_lens[s] - (p.cu_q[s + 1] - row);   // position of this query token
  const int* table = p.block_tables + static_cast<size_t>(s) * p.max_blocks;
  int first = (p.window > 0 && pos + 1 > p.window) ? pos + 1 - p.window : 0;
  if (p.chunk > 0) first = max(first, pos / p.chunk * p.chunk);
  const float r1 = p.r1 != nullptr ? p.r1[h] : 0.f, r2 = p.r1 != nullptr ? p.r2[h] : 0.f;
  const T* kp = static_cast<const T*>(p.k_pool);
  const T* vp = static_cast<const T*>(p.v_pool);
  const bool vec = p.Dk % 4 == 0 && p.ldk % 4 == 0;
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(row) * p.out_stride + static_cast<size_t>(h) * p.Dv;
  const int n_means = p.mean_of > 0 ? first / p.mean_of : 0, n_keys = n_means + pos + 1 - first;   // the means come first
  for (int map = 0; map < p.maps; ++map) {
  const T* q = static_cast<const T*>(p.q) + static_cast<size_t>(row) * p.q_stride + (static_cast<size_t>(h) * p.maps + map) * p.Dk;
  __syncthreads();                                       // (the previous map's results have been read)
  for (int i = threadIdx.x; i < p.Dk; i += blockDim.x) q_s[i] = to_f(q[i]);
  __syncthreads();
  float m = -INFINITY, l = 0.f, acc[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) acc[i] = 0.f;
  for (int c0 = warp * 32; c0 < n_keys; c0 += kAaWarps * 32) {
    const int i0 = c0 + lane, key = first + i0 - n_means;
    const bool ok = i0 < n_keys;
    float sc = -INFINITY;
    long long prow = 0;                                  // pool row; ~row of the means
    if (ok) {
      const T* kr;
      if (i0 < n_means) {
        const int page = ((i0 + 1) * p.mean_of - 1) / p.block_size;
        const long long m = (static_cast<long long>(table[page]) * p.Hkv + hk) * p.mean_rows + i0 - page * p.block_size / p.mean_of;
        kr = static_cast<const T*>(p.k_mean) + m * p.ldk;
        prow = ~m;
      } else {
        prow = (static_cast<long long>(table[key / p.block_size]) * p.Hkv + hk) * p.block_size + key % p.block_size;
        kr = kp + prow * p.ldk + map * p.Dk;
      }
      float d = 0.f;
      if (vec) {
        float e[4] = {0.f, 0.f, 0.f, 0.f};
        for (int i = 0; i < p.Dk; i += 4) {
          float f[4];
          load_v<4>(kr + i, f);
#pragma unroll
          for (int c = 0; c < 4; ++c) e[c] = fmaf(f[c], q_s[i + c], e[c]);
        }
        d = (e[0] + e[1]) + (e[2] + e[3]);
      } else {
        for (int i = 0; i < p.Dk; ++i) d = fmaf(to_f(kr[i]), q_s[i], d);
      }
      sc = d * p.scale;
      if (p.softcap > 0.f) sc = p.softcap * tanhf(sc / p.softcap);
      if (p.r1 != nullptr) sc -= r1 * log1pf(r2 * static_cast<float>(pos - key));
    }
    const float mn = fmaxf(m, warp_max(sc));
    const float pr = ok ? expf(sc - mn) : 0.f;
    const float corr = m > -INFINITY ? expf(m - mn) : 0.f;
    l = l * corr + warp_sum(pr);
    m = mn;
#pragma unroll
    for (int i = 0; i < NV; ++i) acc[i] *= corr;
    const int nk = min(32, n_keys - c0);
    for (int t = 0; t < nk; ++t) {
      const float pt = __shfl_sync(0xffffffffu, pr, t);
      const long long vrow = __shfl_sync(0xffffffffu, prow, t);
      const T* vr = vrow >= 0 ? vp + vrow * p.ldv : static_cast<const T*>(p.v_mean) + ~vrow * p.ldv;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = lane + 32 * i;
        if (d < p.Dv) acc[i] = fmaf(pt, to_f(vr[d]), acc[i]);
      }
    }
  }
  if (lane == 0) m_s[warp] = m, l_s[warp] = l;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = lane + 32 * i;
    if (d < p.Dv) o_s[warp * p.Dv + d] = acc[i];
  }
  __syncthreads();
  float mm = p.sinks != nullptr ? p.sinks[h] : -INFINITY;
#pragma unroll
  for (int w = 0; w < kAaWarps; ++w) mm = fmaxf(mm, m_s[w]);
  float den = p.sinks != nullptr ? expf(p.sinks[h] - mm) : 0.f, f[kAaWarps];
#pragma unroll
  for (int w = 0; w < kAaWarps; ++w) {
    f[w] = m_s[w] > -INFINITY ? expf(m_s[w] - mm) : 0.f;
    den += l_s[w] * f[w];
  }
  const T* gate = p.gate == nullptr ? nullptr
                                    : static_cast<const T*>(p.gate) + static_cast<size_t>(row) * p.gate_stride + static_cast<size_t>(h) * p.Dv;
  for (int d = threadIdx.x; d < p.Dv; d += blockDim.x) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < kAaWarps; ++w) o += o_s[w * p.Dv + d] * f[w];
    o = den > 0.f ? o / den : 0.f;
    if (p.maps == 2) {                                   // (a thread meets the same columns in both maps)
      a_s[d] = map == 0 ? o : a_s[d] - p.lambda * o;
      continue;
    }
    if (gate != nullptr) o *= sigmoid_f(to_f(gate[d]));
    out[d] = from_f<T>(o * p.gain);
  }
  }
  if (p.maps != 2) return;
  float ss[1] = {0.f};
  for (int d = threadIdx.x; d < p.Dv; d += blockDim.x) ss[0] += a_s[d] * a_s[d];
  block_sums<1>(ss, red);
  const float r = p.gain / sqrtf(ss[0] / p.Dv + p.eps);
  for (int d = threadIdx.x; d < p.Dv; d += blockDim.x) out[d] = from_f<T>(a_s[d] * r);
}

template <typename T>
static int launch_attention_any(const AnyAttnParams& p, int rows, cudaStream_t st) {
  const dim3 grid(rows, p.Hq), block(kAaWarps * 32);
  const size_t smem = (static_cast<size_t>(p.Dk) + (kAaWarps + (p.maps == 2 ? 1 : 0)) * static_cast<size_t>(p.Dv)) * sizeof(float);
  if (smem > 40 * 1024) return -1;
  if (p.Dv <= 64) return static_cast<int>(launch_kernel(attention_any_kernel<T, 2>, grid, block, smem, st, p));
  if (p.Dv <= 128) return static_cast<int>(launch_kernel(attention_any_kernel<T, 4>, grid, block, smem, st, p));
  if (p.Dv <= 256) return static_cast<int>(launch_kernel(attention_any_kernel<T, 8>, grid, block, smem, st, p));
  if (p.Dv <= 1024) return static_cast<int>(launch_kernel(attention_any_kernel<T, 32>, grid, block, smem, st, p));
  return -1;
}

}  // namespace mx

using namespace mx;

static int gemm_any(const void* x, const void* w, void* out, const void* bias, const void* residual, int M, int N, int K,
                    long long ldx, long long ldw, long long ldo, long long ldr, int batch, long long bx, long long bw, long long bo,
                    int fp32, int out_fp32, void* stream) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  const int gy = (M + kGaTile - 1) / kGaTile;
  if (K <= 0 || gy > 65535 || batch > 65535) return -1;
  const dim3 grid((N + kGaTile - 1) / kGaTile, gy, batch), block(kGaThreads);
  auto st = static_cast<cudaStream_t>(stream);
#define MX_GA(T, TO)                                                                                                   \
  return static_cast<int>(launch_kernel(gemm_any_kernel<T, TO>, grid, block, 0, st, static_cast<const T*>(x),         \
                                        static_cast<const T*>(w), static_cast<TO*>(out), static_cast<const T*>(bias), \
                                        static_cast<const T*>(residual), M, N, K, ldx, ldw, ldo, ldr, bx, bw, bo))
  if (fp32) MX_GA(float, float);
  if (out_fp32) MX_GA(__nv_bfloat16, float);
  MX_GA(__nv_bfloat16, __nv_bfloat16);
#undef MX_GA
}

// fp32: operands fp32 (else bf16); out_fp32: result fp32 (implied by fp32 operands).
extern "C" int mx_gemm_any(const void* x, const void* w, void* out, const void* bias, const void* residual, int M, int N,
                           int K, long long ldx, long long ldw, long long ldo, long long ldr, int fp32, int out_fp32,
                           void* stream) {
  return gemm_any(x, w, out, bias, residual, M, N, K, ldx, ldw, ldo, ldr, 1, 0, 0, 0, fp32, out_fp32, stream);
}

// `batch` products whose operands and results lie bx / bw / bo elements apart.
extern "C" int mx_batched_gemm_any(const void* x, const void* w, void* out, int batch, int M, int N, int K, long long ldx,
                                   long long ldw, long long ldo, long long bx, long long bw, long long bo, int fp32,
                                   void* stream) {
  return gemm_any(x, w, out, nullptr, nullptr, M, N, K, ldx, ldw, ldo, 0, batch, bx, bw, bo, fp32, 0, stream);
}

// out [list rows, N]; w [E, N, K]; at most max_rows rows per expert.
extern "C" int mx_grouped_gemm_any(const void* x, const void* w, void* out, const int* offsets, const int* row_map, int E, int max_rows,
                                   int N, int K, long long ldx, int fp32, void* stream) {
  if (E <= 0 || N <= 0 || max_rows <= 0) return 0;
  const int gy = (max_rows + kGaTile - 1) / kGaTile;
  if (K <= 0 || gy > 65535 || E > 65535) return -1;
  const dim3 grid((N + kGaTile - 1) / kGaTile, gy, E), block(kGaThreads);
  auto st = static_cast<cudaStream_t>(stream);
#define MX_GG(T)                                                                                                       \
  return static_cast<int>(launch_kernel(grouped_gemm_any_kernel<T>, grid, block, 0, st, static_cast<const T*>(x),     \
                                        static_cast<const T*>(w), static_cast<T*>(out), offsets, row_map, N, K, ldx))
  if (fp32) MX_GG(float);
  MX_GG(__nv_bfloat16);
#undef MX_GG
}

// Query row r of sequence s (cu_q[s] <= r < cu_q[s + 1]) is token context_lens[s] - (cu_q[s + 1] - r) of
// its sequence. r1 / r2, sinks, gate may be NULL. Pools hold the activation type. maps == 2: differential heads (Dk columns of
// a query and key head are both maps; no sinks, bias or gate), else gain multiplies the result. Output rows are out_stride
// elements apart. mean_of > 0 (with a window; one map, no chunks, no bias): block means.
extern "C" int mx_paged_attention_any(const void* q, long long q_stride, const void* k_pool, const void* v_pool,
                                      const void* block_tables, const void* cu_q, const void* context_lens,
                                      const void* sinks, const void* r1, const void* r2, const void* gate,
                                      long long gate_stride, void* out, long long out_stride, int num_seqs, int rows, int Hq,
                                      int Hkv, int Dk, int Dv, int ldk, int ldv, int block_size, int max_blocks, int window,
                                      int chunk, float scale, float softcap, int maps, float lambda, float gain, float eps,
                                      const void* k_mean, const void* v_mean, int mean_of, int fp32, void* stream) {
  if (num_seqs <= 0 || rows <= 0) return 0;
  if (mean_of > 0 && (window <= 0 || chunk > 0 || maps != 1 || r1 != nullptr || k_mean == nullptr || v_mean == nullptr)) return -1;
  if ((maps != 1 && maps != 2) || (maps == 2 && (Dk % 2 || sinks != nullptr || r1 != nullptr || gate != nullptr))) return -1;
  if (Hkv <= 0 || Hq % Hkv || Hq > 65535 || Dk <= 0 || Dv <= 0 || ldk < Dk || ldv < Dv ||
      (r1 == nullptr) != (r2 == nullptr))
    return -1;
  AnyAttnParams p{q, q_stride, k_pool, v_pool, static_cast<const int*>(block_tables), static_cast<const int*>(cu_q),
                  static_cast<const int*>(context_lens), static_cast<const float*>(sinks), static_cast<const float*>(r1),
                  static_cast<const float*>(r2), gate, gate_stride, out, num_seqs, Hq, Hkv, Dk / maps, Dv, ldk, ldv,
                  block_size, max_blocks, window, chunk, scale, softcap, maps, lambda, gain, eps, out_stride, k_mean, v_mean,
                  mean_of, mean_of > 0 ? (block_size + mean_of - 1) / mean_of : 0};
  auto st = static_cast<cudaStream_t>(stream);
  return fp32 ? launch_attention_any<float>(p, rows, st) : launch_attention_any<__nv_bfloat16>(p, rows, st);
}
