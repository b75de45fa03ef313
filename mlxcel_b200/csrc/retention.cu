// Retention: linear attention with a fixed decay per head, no softmax and no denominator.
//   q, k rotated by the token's position (dimension i turns with i + rot / 2, the rest passes), k times D^(-1/2) behind it
//   S <- decay S + k v^T;  o = S^T q;  out = o / rms(o) * silu(gate) * gain
// State [slots, H, D, V] fp32; everything behind the projections is fp32.
//
// Kernels:
//   retention_step   pieces of one token (decode): one CTA per (head, row); rotation, recurrence, norm and gate fused, the state
//                    streams through registers once
//   retention_chunks (retention_tc.cu)   longer pieces, bf16: chunks of 128 tokens on the tensor cores
//   retention_prep / retention_scan / retention_post   the same for fp32 and other sizes: rotation of all tokens at once into
//                    zero-padded fp32 rows; the recurrence with the state in registers, two channels per packed fp32
//                    instruction; norm and gate
#include "api.h"
#include "retention.cuh"

namespace mx {

__device__ __forceinline__ float ret_silu(float x) { return x * sigmoid_f(x); }

// ----------------------------------------------------------------------------- one token per piece
constexpr int kRsThreads = 256;

// W: columns of a thread's access. Threads tile the state as (phase, column group): phase f takes rows f, f + phases, ..
template <typename T, int W>
__global__ void __launch_bounds__(kRsThreads) retention_step_kernel(const RetentionParams p) {
  extern __shared__ __align__(16) float rs_smem[];
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const int D = p.D, V = p.V, h = blockIdx.x, j = blockIdx.y, tid = threadIdx.x;
  const int t = p.cu[j], slot = p.slots[j];
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(t) * p.ldo + static_cast<size_t>(h) * V;
  if (slot < 0) {
    for (int i = tid; i < V; i += kRsThreads) out[i] = from_f<T>(0.f);
    return;
  }
  float *q_s = rs_smem, *k_s = q_s + D, *part = k_s + D + (-2 * D & 3);      // part: [phases][V]
  const T* row = static_cast<const T*>(p.proj) + static_cast<size_t>(t) * p.ld;
  const T *qr = row + h * D, *kr = row + (p.H + h) * D, *vr = row + 2 * p.H * D + h * V, *gr = vr + p.H * V;
  const float ks = rsqrtf(static_cast<float>(D)), pos = static_cast<float>(p.positions[t]);
  const int half = p.rot / 2;
  for (int i = tid; i < D; i += kRsThreads) {
    if (i < half) {
      float s, c;
      sincosf(pos * p.inv_freq[i], &s, &c);
      const float qu = to_f(qr[i]), qv = to_f(qr[i + half]), ku = to_f(kr[i]), kv = to_f(kr[i + half]);
      q_s[i] = qu * c - qv * s, q_s[i + half] = qv * c + qu * s;
      k_s[i] = (ku * c - kv * s) * ks, k_s[i + half] = (kv * c + ku * s) * ks;
    } else if (i >= p.rot) {
      q_s[i] = to_f(qr[i]), k_s[i] = to_f(kr[i]) * ks;
    }
  }
  __syncthreads();
  const bool fresh = p.reset[j] != 0;
  const float g = p.decay[h];
  float* S = p.memory + (static_cast<size_t>(slot) * p.H + h) * D * V;
  const int groups = V / W, cols = min(groups, kRsThreads), phases = kRsThreads / cols, phase = tid / cols;
  if (phase < phases)
    for (int cg = tid - phase * cols; cg < groups; cg += cols) {
      float v[W], o[W];
      load_v<W>(vr + cg * W, v);
#pragma unroll
      for (int e = 0; e < W; ++e) o[e] = 0.f;
      constexpr int B = 8;                                 // state rows requested at a time
      for (int i0 = phase; i0 < D; i0 += B * phases) {
        float s[B][W];
#pragma unroll
        for (int b = 0; b < B; ++b) {
          const int i = i0 + b * phases;
          if (i < D && !fresh) load_v<W>(S + static_cast<size_t>(i) * V + cg * W, s[b]);
          else {
#pragma unroll
            for (int e = 0; e < W; ++e) s[b][e] = 0.f;
          }
        }
#pragma unroll
        for (int b = 0; b < B; ++b) {
          const int i = i0 + b * phases;
          if (i >= D) break;
          const float a = k_s[i], c = q_s[i];
#pragma unroll
          for (int e = 0; e < W; ++e) {
            s[b][e] = fmaf(a, v[e], g * s[b][e]);
            o[e] = fmaf(c, s[b][e], o[e]);
          }
          store_v<W>(S + static_cast<size_t>(i) * V + cg * W, s[b]);
        }
      }
#pragma unroll
      for (int e = 0; e < W; ++e) part[static_cast<size_t>(phase) * V + cg * W + e] = o[e];
    }
  __syncthreads();
  float ss[1] = {0.f};
  for (int c = tid; c < V; c += kRsThreads) {
    float o = 0.f;
    for (int f = 0; f < phases; ++f) o += part[static_cast<size_t>(f) * V + c];
    part[c] = o;                                           // (column c is this thread's alone)
    ss[0] = fmaf(o, o, ss[0]);
  }
  block_sums<1>(ss, red);
  const float r = p.gain / sqrtf(ss[0] / V + p.norm_eps);
  for (int c = tid; c < V; c += kRsThreads) out[c] = from_f<T>(part[c] * r * ret_silu(to_f(gr[c])));
}

// ----------------------------------------------------------------------------- longer pieces
// One CTA per token: the angles once, then all heads.
template <typename T>
__global__ void __launch_bounds__(256) retention_prep_kernel(const RetentionParams p, float* __restrict__ scratch, int row0, int N) {
  extern __shared__ float rp_cs[];                         // [rot / 2] cosines, then sines
  pdl_trigger();
  pdl_wait();
  const int n = blockIdx.x, t = row0 + n, D = p.D, V = p.V, H = p.H, half = p.rot / 2, DP = ret_dp(D), VP = ret_vp(V);
  const float pos = static_cast<float>(p.positions[t]), ks = rsqrtf(static_cast<float>(D));
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * p.inv_freq[i], &rp_cs[half + i], &rp_cs[i]);
  __syncthreads();
  const RetentionScratch sc = ret_scratch(scratch, N, H, D, V);
  const T* row = static_cast<const T*>(p.proj) + static_cast<size_t>(t) * p.ld;
  for (int i = threadIdx.x; i < 2 * H * DP; i += blockDim.x) {
    const int hd = i / DP, d = i - hd * DP;                // heads of q, then of k
    float f = 0.f;
    if (d < D) {
      const T* src = row + static_cast<size_t>(hd) * D;
      const float a = to_f(src[d]);
      f = d < half ? a * rp_cs[d] - to_f(src[d + half]) * rp_cs[half + d] : d < p.rot ? a * rp_cs[d - half] + to_f(src[d - half]) * rp_cs[d] : a;
      if (hd >= H) f *= ks;
    }
    (hd < H ? sc.q + (static_cast<size_t>(n) * H + hd) * DP : sc.k + (static_cast<size_t>(n) * H + hd - H) * DP)[d] = f;
  }
  const T* vr = row + 2 * H * D;
  for (int i = threadIdx.x; i < H * VP; i += blockDim.x) {
    const int hd = i / VP, d = i - hd * VP;
    sc.v[static_cast<size_t>(n) * H * VP + i] = d < V ? to_f(vr[hd * V + d]) : 0.f;
  }
}

using ret2 = unsigned long long;                           // a packed pair of fp32
__device__ __forceinline__ ret2 ret_pack(float a, float b) {
  ret2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void ret_unpack(ret2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ ret2 ret_fma(ret2 a, ret2 b, ret2 c) {
  ret2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ ret2 ret_mul(ret2 a, ret2 b) {
  ret2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ void ret_copy16(float* smem, const float* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}

// Eight lanes share COLS neighbouring columns of one head's state; a lane keeps RPT key channels of each (4 l .. 4 l + 3, then 32
// further on) as packed pairs. The vectors of TOK tokens are double-buffered. Per token: the update, one partial dot per column
// with q, and a halving exchange over the lanes (the two low lane bits end with a column of their own).
constexpr int kRcThreads = 64;

template <int RPT, int COLS>
__global__ void __launch_bounds__(kRcThreads) retention_scan_kernel(const RetentionParams p, float* __restrict__ scratch, int row0, int N) {
  constexpr int DP = 8 * RPT, P2 = RPT / 2, CTA = kRcThreads / 8 * COLS, TOK = RPT <= 16 ? 8 : 4, STAGE = TOK * (2 * DP + CTA);
  static_assert(COLS == 4 || COLS == 2, "columns of a lane");
  extern __shared__ __align__(16) float rc_smem[];
  pdl_trigger();
  pdl_wait();
  const int D = p.D, V = p.V, H = p.H, VP = ret_vp(V), cbs = VP / CTA;
  const int h = blockIdx.x / cbs, cb = blockIdx.x - h * cbs, j = blockIdx.y;
  const int t0 = p.cu[j] - row0, t1 = p.cu[j + 1] - row0, slot = p.slots[j];
  if (t1 <= t0) return;
  const RetentionScratch sc = ret_scratch(scratch, N, H, D, V);
  const int lane = threadIdx.x & 31, l8 = lane & 7;
  if (slot < 0) {
    for (int i = threadIdx.x; i < (t1 - t0) * CTA; i += kRcThreads)
      sc.o[(static_cast<size_t>(t0 + i / CTA) * H + h) * VP + cb * CTA + i % CTA] = 0.f;
    return;
  }
  const bool fresh = p.reset[j] != 0;
  const int c_in = (threadIdx.x >> 3) * COLS, col0 = cb * CTA + c_in;
  const auto chan = [&](int r) { return (r >> 2) * 32 + 4 * l8 + (r & 3); };
  float* S = p.memory + (static_cast<size_t>(slot) * H + h) * D * V;
  ret2 s[P2][COLS];
#pragma unroll
  for (int r = 0; r < P2; ++r)
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
      const int a = chan(2 * r), col = col0 + c;
      const bool in = col < V && !fresh;
      s[r][c] = ret_pack(in && a < D ? S[static_cast<size_t>(a) * V + col] : 0.f, in && a + 1 < D ? S[static_cast<size_t>(a + 1) * V + col] : 0.f);
    }
  const auto load = [&](int c0, int buf) {
    float* st = rc_smem + buf * STAGE;
    const int nt = min(TOK, t1 - c0);
    constexpr int QK = DP / 4, VC = CTA / 4, PER = 2 * QK + VC;      // 16-byte groups of a token
    for (int i = threadIdx.x; i < nt * PER; i += kRcThreads) {
      const int t = i / PER, g = i - t * PER;
      const size_t n = static_cast<size_t>(c0 + t) * H + h;
      const float* src = g < QK ? sc.k + n * DP + 4 * g : g < 2 * QK ? sc.q + n * DP + 4 * (g - QK) : sc.v + n * VP + cb * CTA + 4 * (g - 2 * QK);
      ret_copy16(st + t * (2 * DP + CTA) + 4 * g, src);
    }
  };
  const float g1 = p.decay[h];
  const ret2 g2 = ret_pack(g1, g1);
  const bool b0 = l8 & 1, b1 = l8 & 2;
  const int own = COLS == 4 ? 2 * b0 + b1 : b0;
  load(t0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  int buf = 0;
  for (int c0 = t0; c0 < t1; c0 += TOK, buf ^= 1) {
    if (c0 + TOK < t1) load(c0 + TOK, buf ^ 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const float* st = rc_smem + buf * STAGE;
    const int nt = min(TOK, t1 - c0);
    float* o = sc.o + (static_cast<size_t>(c0) * H + h) * VP + col0 + own;
    for (int t = 0; t < nt; ++t, st += 2 * DP + CTA, o += static_cast<size_t>(H) * VP) {
      ret2 dot[COLS], v2[COLS];
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        const float v = st[2 * DP + c_in + c];
        v2[c] = ret_pack(v, v);
        dot[c] = 0ull;
      }
#pragma unroll
      for (int r = 0; r < P2; r += 2) {
        const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(st + r * 16 + 4 * l8), q = *reinterpret_cast<const ulonglong2*>(st + DP + r * 16 + 4 * l8);
#pragma unroll
        for (int c = 0; c < COLS; ++c) {
          s[r][c] = ret_fma(k.x, v2[c], ret_mul(g2, s[r][c]));
          s[r + 1][c] = ret_fma(k.y, v2[c], ret_mul(g2, s[r + 1][c]));
          dot[c] = ret_fma(q.x, s[r][c], dot[c]);
          dot[c] = ret_fma(q.y, s[r + 1][c], dot[c]);
        }
      }
      float x[COLS];
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        float a, b;
        ret_unpack(dot[c], a, b);
        x[c] = a + b;
      }
      float y;
      if constexpr (COLS == 4) {
        const float y0 = (b0 ? x[2] : x[0]) + __shfl_xor_sync(0xffffffffu, b0 ? x[0] : x[2], 1);
        const float y1 = (b0 ? x[3] : x[1]) + __shfl_xor_sync(0xffffffffu, b0 ? x[1] : x[3], 1);
        y = (b1 ? y1 : y0) + __shfl_xor_sync(0xffffffffu, b1 ? y0 : y1, 2);
      } else {
        y = (b0 ? x[1] : x[0]) + __shfl_xor_sync(0xffffffffu, b0 ? x[0] : x[1], 1);
        y += __shfl_xor_sync(0xffffffffu, y, 2);
      }
      y += __shfl_xor_sync(0xffffffffu, y, 4);
      if (l8 < COLS) *o = y;
    }
    __syncthreads();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int r = 0; r < P2; ++r)
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
      const int a = chan(2 * r), col = col0 + c;
      float lo, hi;
      ret_unpack(s[r][c], lo, hi);
      if (col < V && a < D) S[static_cast<size_t>(a) * V + col] = lo;
      if (col < V && a + 1 < D) S[static_cast<size_t>(a + 1) * V + col] = hi;
    }
}

// One warp per (token, head): o / rms(o) * silu(gate) * gain. Rows of o are ret_vp(V) wide, zero from V on.
template <typename T>
__global__ void __launch_bounds__(256) retention_post_kernel(const RetentionParams p, const float* __restrict__ rows_o, int row0, int N) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, V = p.V, VP = ret_vp(V);
  const unsigned gw = blockIdx.x * (blockDim.x / 32) + (threadIdx.x >> 5);
  if (gw >= static_cast<unsigned>(N) * p.H) return;
  const int n = static_cast<int>(gw / p.H), h = static_cast<int>(gw - static_cast<unsigned>(n) * p.H);
  const float* o = rows_o + (static_cast<size_t>(n) * p.H + h) * VP;
  const T* z = static_cast<const T*>(p.proj) + static_cast<size_t>(row0 + n) * p.ld + 2 * p.H * p.D + p.H * V + h * V;
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(row0 + n) * p.ldo + static_cast<size_t>(h) * V;
  float s = 0.f;
  for (int c = 4 * lane; c < VP; c += 128) {               // (padding columns are zero)
    float a[4];
    load_v<4>(o + c, a);
#pragma unroll
    for (int e = 0; e < 4; ++e) s = fmaf(a[e], a[e], s);
  }
  const float r = p.gain / sqrtf(warp_sum(s) / V + p.norm_eps);
  const size_t group = sizeof(T) * 4;
  if (V % 4 == 0 && reinterpret_cast<uintptr_t>(z) % group == 0 && reinterpret_cast<uintptr_t>(out) % group == 0) {
    for (int c = 4 * lane; c < V; c += 128) {
      float a[4], g[4];
      load_v<4>(o + c, a);
      load_v<4>(z + c, g);
#pragma unroll
      for (int e = 0; e < 4; ++e) a[e] *= r * ret_silu(g[e]);
      store_v<4>(out + c, a);
    }
    return;
  }
  for (int c = lane; c < V; c += 32) out[c] = from_f<T>(o[c] * r * ret_silu(to_f(z[c])));
}

template <int RPT, int COLS>
static int launch_retention_scan(const RetentionParams& p, float* scratch, int pieces, int row0, int N, cudaStream_t st) {
  constexpr int CTA = kRcThreads / 8 * COLS, smem = 2 * (RPT <= 16 ? 8 : 4) * (2 * 8 * RPT + CTA) * 4;
  static_assert(smem <= 48 * 1024, "fits the default limit");
  return static_cast<int>(launch_kernel(retention_scan_kernel<RPT, COLS>, dim3(p.H * (ret_vp(p.V) / CTA), pieces), dim3(kRcThreads), smem, st, p,
                                        scratch, row0, N));
}

template <typename T>
static int launch_retention_post(const RetentionParams& p, const float* o, int row0, int N, cudaStream_t st) {
  const long long warps = static_cast<long long>(N) * p.H;
  if (warps > 0x7fffffffll) return -1;
  return static_cast<int>(launch_kernel(retention_post_kernel<T>, dim3(static_cast<unsigned>((warps + 7) / 8)), dim3(256), 0, st, p, o, row0, N));
}

template <typename T>
static int retention_typed(RetentionParams p, int pieces, int n_short, int rows, float* scratch, int form, int* status, cudaStream_t st) {
  if (n_short > 0) {
    const bool vec = p.V % 4 == 0 && p.ld % 4 == 0 && 2 * p.H * p.D % 4 == 0 && aligned_to(p.proj, sizeof(T) * 4) && aligned_to(p.memory, 16);
    const int groups = p.V / (vec ? 4 : 1), cols = groups < kRsThreads ? groups : kRsThreads;
    const size_t smem = (2 * static_cast<size_t>(p.D) + 4 + static_cast<size_t>(kRsThreads / cols) * p.V) * sizeof(float);
    if (smem > 40 * 1024) return -1;
    const dim3 grid(p.H, n_short), block(kRsThreads);
    const int rc = vec ? static_cast<int>(launch_kernel(retention_step_kernel<T, 4>, grid, block, smem, st, p))
                       : static_cast<int>(launch_kernel(retention_step_kernel<T, 1>, grid, block, smem, st, p));
    if (rc) return rc;
  }
  const int np = pieces - n_short, N = rows - n_short;
  if (np <= 0 || N <= 0) return 0;
  if (scratch == nullptr || !aligned_to(scratch, 16)) return -1;
  p.slots += n_short, p.cu += n_short, p.reset += n_short, p.pieces = np;
  if (sizeof(T) == 2 && form == 0 && ret_chunk_covered(p.D, p.V, p.rot)) {
    if (!aligned_to(p.proj, 16) || p.ld % 8 || !aligned_to(p.out, 16) || p.ldo % 8) return -1;
    float* o = p.V > kRetTile ? scratch + static_cast<long long>(N) * p.rot : nullptr;
    const int rc = launch_retention_chunks(p, scratch, o, np, n_short, N, status, st);
    return rc || o == nullptr ? rc : launch_retention_post<T>(p, o, n_short, N, st);
  }
  int rc = static_cast<int>(launch_kernel(retention_prep_kernel<T>, dim3(N), dim3(256), static_cast<size_t>(p.rot) * 4, st, p, scratch, n_short, N));
  if (rc) return rc;
  const int dp = ret_dp(p.D);
  // columns of a lane: two while that leaves every SM no more than one CTA
  const bool few = static_cast<long long>(np) * p.H * (ret_vp(p.V) / 16) <= 148;
  if (dp == 32) rc = few ? launch_retention_scan<4, 2>(p, scratch, np, n_short, N, st) : launch_retention_scan<4, 4>(p, scratch, np, n_short, N, st);
  else if (dp == 64) rc = few ? launch_retention_scan<8, 2>(p, scratch, np, n_short, N, st) : launch_retention_scan<8, 4>(p, scratch, np, n_short, N, st);
  else if (dp == 128) rc = few ? launch_retention_scan<16, 2>(p, scratch, np, n_short, N, st) : launch_retention_scan<16, 4>(p, scratch, np, n_short, N, st);
  else if (dp == 256) rc = launch_retention_scan<32, 2>(p, scratch, np, n_short, N, st);
  else rc = launch_retention_scan<64, 2>(p, scratch, np, n_short, N, st);
  if (rc) return rc;
  return launch_retention_post<T>(p, ret_scratch(scratch, N, p.H, p.D, p.V).o, n_short, N, st);
}

}  // namespace mx

using namespace mx;

extern "C" int mx_retention_chunk_covered(int D, int V, int rot) { return ret_chunk_covered(D, V, rot) ? 1 : 0; }

// form 0: bf16 pieces of covered sizes (mx_retention_chunk_covered) run in chunks; 1: token by token.
extern "C" long long mx_retention_scratch_floats(int tokens, int H, int D, int V, int rot, int bf16, int form) {
  if (bf16 && form == 0 && ret_chunk_covered(D, V, rot)) return ret_chunk_floats(tokens, H, V, rot) + 4;
  return static_cast<long long>(tokens) * H * (2ll * ret_dp(D) + 2ll * ret_vp(V));
}

// A ragged batch of pieces (token rows cu[j] .. cu[j + 1] - 1 of proj, positions and out, state slot slots[j], reset[j] starts from
// zero). The first n_short pieces hold exactly one token each; rows is the total number of token rows. D at most 512.
// scratch: mx_retention_scratch_floats(rows - n_short, ...) floats, or NULL when every piece is short. The chunked form needs proj and out
// aligned to 16 bytes with row strides of whole 16-byte groups.
extern "C" int mx_retention(const void* proj, long long ld, const void* positions, const void* inv_freq, const void* decay, void* memory,
                            const void* slots, const void* cu, const void* reset, void* out, long long ldo, void* scratch, int pieces,
                            int n_short, int rows, int H, int D, int V, int rot, float norm_eps, float gain, int fp32, int form, void* status,
                            void* stream) {
  if (pieces <= 0 || rows <= 0) return 0;
  if (H <= 0 || D <= 0 || D > 512 || V <= 0 || rot < 0 || rot > D || rot % 2 || pieces > 65535 || n_short < 0 || n_short > pieces) return -1;
  RetentionParams p{proj, ld, static_cast<const int*>(positions), static_cast<const float*>(inv_freq), static_cast<const float*>(decay),
                    static_cast<float*>(memory), static_cast<const int*>(slots), static_cast<const int*>(cu), static_cast<const int*>(reset), out, ldo,
                    H, D, V, rot, pieces, norm_eps, gain};
  auto st = static_cast<cudaStream_t>(stream);
  auto* sc = static_cast<float*>(scratch);
  auto* sw = static_cast<int*>(status);
  return fp32 ? retention_typed<float>(p, pieces, n_short, rows, sc, form, sw, st)
              : retention_typed<__nv_bfloat16>(p, pieces, n_short, rows, sc, form, sw, st);
}
