// Gated delta rule with one decay per head, a short causal convolution in front and a gated norm behind.
//   y = silu(conv(x)) per channel of q | k | v;  q = unit(y_q) D^-1/2, k = unit(y_k), unit(z) = z / sqrt(|z|^2 + unit_eps)
//   g = exp(-exp(A_log) softplus(a + dt_bias)), beta = sigmoid(b)
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   out = o / rms(o) * norm_w * silu(gate)
// H value heads share G q/k heads (head h uses h / (H / G)). State [slots, H, D, V] and convolution tail [slots, taps - 1,
// channels] fp32; everything behind the projections is fp32.
//
// The read-out needs the old state only: u = beta (v - g S_old^T k), o = g S_old^T q + (q . k) u, so a token is one pass of two
// dot products per state column, one reduction round and one update.
//
// Kernels:
//   gated_step   pieces of one token (decode): one CTA per (q/k head, row), convolution, rates, recurrence, norm and gate fused;
//                the state passes through registers once
//   gated_prep / gated_scan / gated_post   longer pieces: convolution, unit vectors and rates of all tokens at once; the
//                recurrence with the state in registers, two channels per packed fp32 instruction; the norm and gate
//   gated_scan_any   the recurrence for any sizes, state in global memory
#include "api.h"
#include "typed.cuh"

namespace mx {

struct GatedParams {
  const void* proj;          // rows q [G D] | k [G D] | v [H V] | gate [H V], ld elements apart
  long long ld;
  const float* rates;        // rows write rate [H] | decay [H]
  const float* conv_w;       // [channels, taps]
  const float* A_log;        // [H]
  const float* dt_bias;      // [H]
  const float* norm_w;       // [V]
  float* memory;
  float* tail;
  const int* slots;          // per piece; a negative slot marks a padding row (its output is zero)
  const int* cu;
  const int* reset;
  void* out;                 // [rows, H V]
  int H, G, D, V, taps, pieces;
  float unit_eps, norm_eps;
};

__device__ __forceinline__ int gd_channels(const GatedParams& p) { return 2 * p.G * p.D + p.H * p.V; }
// (within two units in the last place of the exponential)
__device__ __forceinline__ float silu_f(float x) { return __fdividef(x, 1.f + __expf(fminf(-x, 80.f))); }

// Decay of a head. Slow heads sit just below one and are multiplied into the state at every token: 1 + expm1 is within half
// a unit in the last place there.
__device__ __forceinline__ float head_decay(const GatedParams& p, int h, float a) {
  const float z = a + p.dt_bias[h];
  const float soft = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
  return 1.f + expm1f(-expf(p.A_log[h]) * soft);
}

// Packed pairs of fp32.
using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float sum2(f32x2 v) {
  float a, b;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
  return a + b;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// Input of channel c at token t of a piece that starts at row t0: a row of proj, the slot's tail before the piece, or zero.
template <typename T>
__device__ __forceinline__ float conv_input(const GatedParams& p, int c, int t, int t0, int slot, bool fresh) {
  if (t >= t0) return to_f(static_cast<const T*>(p.proj)[static_cast<size_t>(t) * p.ld + c]);
  if (fresh || slot < 0) return 0.f;
  return p.tail[(static_cast<size_t>(slot) * (p.taps - 1) + (p.taps - 1 + t - t0)) * gd_channels(p) + c];
}

// ----------------------------------------------------------------------------- one token per piece
// 8 warps; warp q holds state rows q, q + 8, ... (RPW of them) and lane c the columns 4c .. 4c + 3 (V % 4 == 0, D and V at
// most 128). The heads of a q/k head follow one another; the first one's state is requested before the convolution.
constexpr int kGsThreads = 256;

template <typename T, int RPW>
__global__ void __launch_bounds__(kGsThreads, 2) gated_step_kernel(const GatedParams p) {
  extern __shared__ __align__(16) float gs_v[];             // [heads of the group][V]
  __shared__ float red[3 * 33];
  __shared__ float k_s[128], q_s[128];
  __shared__ __align__(16) float u_s[128];
  __shared__ __align__(16) float part[8][2][128];
  pdl_trigger();
  pdl_wait();
  const int D = p.D, V = p.V, grp = blockIdx.x, j = blockIdx.y, per = p.H / p.G;
  const int t = p.cu[j], slot = p.slots[j], tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(t) * p.H * V + static_cast<size_t>(grp) * per * V;
  if (slot < 0) {
    for (int i = tid; i < per * V; i += kGsThreads) out[i] = from_f<T>(0.f);
    return;
  }
  const bool fresh = p.reset[j] != 0, col_ok = 4 * lane < V;
  float* S = p.memory + (static_cast<size_t>(slot) * p.H + static_cast<size_t>(grp) * per) * D * V;
  float4 st[RPW];
  const auto load_state = [&](int hh) {
#pragma unroll
    for (int q = 0; q < RPW; ++q) {
      const int i = warp + 8 * q;
      st[q] = (col_ok && i < D && !fresh) ? *reinterpret_cast<const float4*>(S + (static_cast<size_t>(hh) * D + i) * V + 4 * lane)
                                          : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load_state(0);
  const int taps = p.taps, ch = gd_channels(p);
  const T* row = static_cast<const T*>(p.proj) + static_cast<size_t>(t) * p.ld;
  float* tail = p.tail + static_cast<size_t>(slot) * (taps - 1) * ch;
  // convolution of one channel; the tail moves up by one
  const auto conv = [&](int c) -> float {
    const float x = to_f(row[c]);
    const float* w = p.conv_w + static_cast<size_t>(c) * taps;
    float y = w[taps - 1] * x;
    for (int i = 0; i < taps - 1; ++i) {
      const float b = fresh ? 0.f : tail[static_cast<size_t>(i) * ch + c];
      y = fmaf(w[i], b, y);
      if (i > 0) tail[static_cast<size_t>(i - 1) * ch + c] = b;
    }
    if (taps > 1) tail[static_cast<size_t>(taps - 2) * ch + c] = x;
    return silu_f(y);
  };
  float s[3] = {0.f, 0.f, 0.f};
  if (tid < 128) {
    if (tid < D) {
      const float q = conv(grp * D + tid);
      q_s[tid] = q;
      s[0] = q * q;
    }
  } else if (tid - 128 < D) {
    const float k = conv((p.G + grp) * D + tid - 128);
    k_s[tid - 128] = k;
    s[1] = k * k;
  }
  for (int i = tid; i < per * V; i += kGsThreads) gs_v[i] = conv(2 * p.G * D + grp * per * V + i);
  block_sums<3>(s, red);
  const float iq = rsqrtf(static_cast<float>(D)) / sqrtf(s[0] + p.unit_eps), ik = 1.f / sqrtf(s[1] + p.unit_eps);
  s[0] = s[1] = s[2] = 0.f;
  if (tid < D) {
    const float q = q_s[tid] * iq, k = k_s[tid] * ik;
    q_s[tid] = q, k_s[tid] = k;
    s[0] = q * k;
  }
  block_sums<3>(s, red);
  const float qk = s[0];
  for (int hh = 0; hh < per; ++hh) {
    const int h = grp * per + hh;
    const float beta = sigmoid_f(p.rates[static_cast<size_t>(t) * 2 * p.H + h]);
    const float g = head_decay(p, h, p.rates[static_cast<size_t>(t) * 2 * p.H + p.H + h]);
    if (hh > 0) load_state(hh);
    float4 ks = make_float4(0.f, 0.f, 0.f, 0.f), qs = ks;
#pragma unroll
    for (int q = 0; q < RPW; ++q) {
      const int i = warp + 8 * q;
      if (i < D) {
        const float a = k_s[i], b = q_s[i];
        ks.x = fmaf(a, st[q].x, ks.x), ks.y = fmaf(a, st[q].y, ks.y), ks.z = fmaf(a, st[q].z, ks.z), ks.w = fmaf(a, st[q].w, ks.w);
        qs.x = fmaf(b, st[q].x, qs.x), qs.y = fmaf(b, st[q].y, qs.y), qs.z = fmaf(b, st[q].z, qs.z), qs.w = fmaf(b, st[q].w, qs.w);
      }
    }
    *reinterpret_cast<float4*>(&part[warp][0][4 * lane]) = ks;
    *reinterpret_cast<float4*>(&part[warp][1][4 * lane]) = qs;
    __syncthreads();
    float o = 0.f;
    if (tid < V) {
      float kk = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) kk += part[w][0][tid], o += part[w][1][tid];
      const float u = beta * (gs_v[hh * V + tid] - g * kk);
      o = g * o + qk * u;
      u_s[tid] = u;
    }
    s[0] = o * o, s[1] = s[2] = 0.f;
    block_sums<3>(s, red);                    // (also publishes u_s; part may be overwritten)
    if (tid < V) {
      const float rs = 1.f / sqrtf(s[0] / V + p.norm_eps);
      const float z = to_f(row[ch + h * V + tid]);
      out[hh * V + tid] = from_f<T>(o * rs * p.norm_w[tid] * silu_f(z));
    }
    if (col_ok) {
      const float4 u4 = *reinterpret_cast<const float4*>(&u_s[4 * lane]);
#pragma unroll
      for (int q = 0; q < RPW; ++q) {
        const int i = warp + 8 * q;
        if (i < D) {
          const float k = k_s[i];
          float4 v;
          v.x = fmaf(k, u4.x, g * st[q].x), v.y = fmaf(k, u4.y, g * st[q].y), v.z = fmaf(k, u4.z, g * st[q].z), v.w = fmaf(k, u4.w, g * st[q].w);
          *reinterpret_cast<float4*>(S + (static_cast<size_t>(hh) * D + i) * V + 4 * lane) = v;
        }
      }
    }
    __syncthreads();                          // u_s of this head has been read
  }
}

// ----------------------------------------------------------------------------- longer pieces
// Scratch of one call over N tokens (rows row0 .. row0 + N - 1), fp32:
//   rates [N, H, 4] (g, beta, q.k, 0) | q [N, G, D] | k [N, G, D] | v [N, H, V] | o [N, H, V]
struct GatedScratch {
  float *rates, *q, *k, *v, *o;
};
__host__ __device__ inline GatedScratch gd_scratch(float* s, long long N, int H, int G, int D, int V) {
  GatedScratch r;
  r.rates = s;
  r.q = r.rates + N * H * 4;
  r.k = r.q + N * G * D;
  r.v = r.k + N * G * D;
  r.o = r.v + N * H * V;
  return r;
}

__device__ __forceinline__ int piece_of(const GatedParams& p, int t) {   // piece j with cu[j] <= t < cu[j + 1]
  int lo = 0, hi = p.pieces;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (p.cu[mid] <= t) lo = mid;
    else hi = mid;
  }
  return lo;
}

constexpr int kGpTok = 16;         // tokens a warp takes
constexpr int kGpBatch = 4;        // of which it requests so many at a time
constexpr int kGpThreads = 128;

// Silu of the convolution of four neighbouring channels over a run of tokens: the taps' inputs slide through registers.
template <typename T, int TAPS>
struct ConvRun {
  const GatedParams& p;
  int c, j, t0, t1;
  float w[TAPS][4], x[TAPS][4];
  __device__ ConvRun(const GatedParams& p_, int c_, int t) : p(p_), c(c_) {
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int i = 0; i < TAPS; ++i) w[i][e] = p.conv_w[static_cast<size_t>(c + e) * TAPS + i];
    enter(piece_of(p, t), t);
  }
  __device__ void enter(int piece, int t) {          // x[1 ..] = the TAPS - 1 inputs before token t
    j = piece, t0 = p.cu[j], t1 = p.cu[j + 1];
    const int slot = p.slots[j];
    const bool fresh = p.reset[j] != 0;
#pragma unroll
    for (int i = 1; i < TAPS; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) x[i][e] = conv_input<T>(p, c + e, t - TAPS + i, t0, slot, fresh);
  }
  __device__ void input(int t, float (&in)[4]) const { load_v<4>(static_cast<const T*>(p.proj) + static_cast<size_t>(t) * p.ld + c, in); }
  __device__ void next(int t, const float (&in)[4], float (&y)[4]) {
    if (t >= t1) {
      int n = j + 1;
      while (p.cu[n + 1] <= t) ++n;
      enter(n, t);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < TAPS; ++i) {
        x[i][e] = i + 1 < TAPS ? x[i + 1 < TAPS ? i + 1 : i][e] : in[e];
        s = fmaf(w[i][e], x[i][e], s);
      }
      y[e] = silu_f(s);
    }
  }
};

__device__ __forceinline__ void write_rates(const GatedParams& p, const GatedScratch& sc, int t, int n, int grp, float qk, int lane) {
  const int per = p.H / p.G;
  for (int i = lane; i < per; i += 32) {
    const int h = grp * per + i;
    const float* r = p.rates + static_cast<size_t>(t) * 2 * p.H;
    *reinterpret_cast<float4*>(sc.rates + (static_cast<size_t>(n) * p.H + h) * 4) =
        make_float4(head_decay(p, h, r[p.H + h]), sigmoid_f(r[h]), qk, 0.f);
  }
}

// A warp takes kGpTok tokens of one unit: units 0 .. G - 1 are the q/k heads, G .. G + H - 1 the value heads. Widths are
// multiples of 4 and at most 128.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kGpThreads)
gated_prep_kernel(const GatedParams p, float* __restrict__ scratch, int row0, int N) {
  pdl_trigger();
  pdl_wait();
  const int unit = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, D = p.D, V = p.V;
  const int n0 = (blockIdx.x * (kGpThreads / 32) + warp) * kGpTok, n1 = min(N, n0 + kGpTok);
  if (n0 >= N) return;
  const GatedScratch sc = gd_scratch(scratch, N, p.H, p.G, D, V);
  const int c = 4 * lane;
  if (unit < p.G) {
    const bool in = c < D;
    ConvRun<T, TAPS> q(p, unit * D + (in ? c : 0), row0 + n0), k(p, (p.G + unit) * D + (in ? c : 0), row0 + n0);
    const float dq = rsqrtf(static_cast<float>(D));
    for (int m0 = n0; m0 < n1; m0 += kGpBatch) {
      float qi[kGpBatch][4], ki[kGpBatch][4];
#pragma unroll
      for (int i = 0; i < kGpBatch; ++i) q.input(row0 + min(m0 + i, n1 - 1), qi[i]), k.input(row0 + min(m0 + i, n1 - 1), ki[i]);
#pragma unroll
      for (int i = 0; i < kGpBatch; ++i) {
        const int n = m0 + i;
        if (n >= n1) break;
        float a[4], b[4];
        q.next(row0 + n, qi[i], a);
        k.next(row0 + n, ki[i], b);
        float aa = 0.f, bb = 0.f, ab = 0.f;
        if (in) {
#pragma unroll
          for (int e = 0; e < 4; ++e) aa = fmaf(a[e], a[e], aa), bb = fmaf(b[e], b[e], bb), ab = fmaf(a[e], b[e], ab);
        }
        aa = warp_sum(aa), bb = warp_sum(bb), ab = warp_sum(ab);
        const float iq = dq / sqrtf(aa + p.unit_eps), ik = 1.f / sqrtf(bb + p.unit_eps);
        if (in) {
#pragma unroll
          for (int e = 0; e < 4; ++e) a[e] *= iq, b[e] *= ik;
          store_v<4>(sc.q + (static_cast<size_t>(n) * p.G + unit) * D + c, a);
          store_v<4>(sc.k + (static_cast<size_t>(n) * p.G + unit) * D + c, b);
        }
        write_rates(p, sc, row0 + n, n, unit, ab * iq * ik, lane);
      }
    }
  } else if (c < V) {
    const int h = unit - p.G;
    ConvRun<T, TAPS> v(p, 2 * p.G * D + h * V + c, row0 + n0);
    for (int m0 = n0; m0 < n1; m0 += kGpBatch) {
      float vi[kGpBatch][4];
#pragma unroll
      for (int i = 0; i < kGpBatch; ++i) v.input(row0 + min(m0 + i, n1 - 1), vi[i]);
#pragma unroll
      for (int i = 0; i < kGpBatch; ++i) {
        const int n = m0 + i;
        if (n >= n1) break;
        float a[4];
        v.next(row0 + n, vi[i], a);
        store_v<4>(sc.v + (static_cast<size_t>(n) * p.H + h) * V + c, a);
      }
    }
  }
}

// The same for any widths and taps: one warp per (token, unit).
template <typename T>
__global__ void __launch_bounds__(kGpThreads)
gated_prep_any_kernel(const GatedParams p, float* __restrict__ scratch, int row0, int N) {
  pdl_trigger();
  pdl_wait();
  const int unit = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, D = p.D, V = p.V;
  const int n = blockIdx.x * (kGpThreads / 32) + warp;
  if (n >= N) return;
  const GatedScratch sc = gd_scratch(scratch, N, p.H, p.G, D, V);
  const int t = row0 + n, j = piece_of(p, t), t0 = p.cu[j], slot = p.slots[j];
  const bool fresh = p.reset[j] != 0;
  const auto conv = [&](int c) -> float {
    float y = 0.f;
    for (int i = 0; i < p.taps; ++i) y = fmaf(p.conv_w[static_cast<size_t>(c) * p.taps + i], conv_input<T>(p, c, t - p.taps + 1 + i, t0, slot, fresh), y);
    return silu_f(y);
  };
  if (unit < p.G) {
    float* q = sc.q + (static_cast<size_t>(n) * p.G + unit) * D;
    float* k = sc.k + (static_cast<size_t>(n) * p.G + unit) * D;
    float aa = 0.f, bb = 0.f, ab = 0.f;
    for (int c = lane; c < D; c += 32) {
      const float a = conv(unit * D + c), b = conv((p.G + unit) * D + c);
      aa = fmaf(a, a, aa), bb = fmaf(b, b, bb), ab = fmaf(a, b, ab);
      q[c] = a, k[c] = b;
    }
    aa = warp_sum(aa), bb = warp_sum(bb), ab = warp_sum(ab);
    const float iq = rsqrtf(static_cast<float>(D)) / sqrtf(aa + p.unit_eps), ik = 1.f / sqrtf(bb + p.unit_eps);
    for (int c = lane; c < D; c += 32) q[c] *= iq, k[c] *= ik;      // (a lane's own columns)
    write_rates(p, sc, t, n, unit, ab * iq * ik, lane);
  } else {
    const int h = unit - p.G;
    for (int c = lane; c < V; c += 32) sc.v[(static_cast<size_t>(n) * p.H + h) * V + c] = conv(2 * p.G * D + h * V + c);
  }
}

// The tail a piece leaves: its last taps - 1 inputs (old tail entries move up where the piece is shorter). Channels of value
// head h, and of its q/k head with the group's first value head.
template <typename T>
__device__ void write_tail(const GatedParams& p, int h, int t0, int t1, int slot, bool fresh) {
  const int per = p.H / p.G, grp = h / per, keep = p.taps - 1, ch = gd_channels(p);
  float* tail = p.tail + static_cast<size_t>(slot) * keep * ch;
  const auto move = [&](int c) {
    for (int i = 0; i < keep; ++i) tail[static_cast<size_t>(i) * ch + c] = conv_input<T>(p, c, t1 - keep + i, t0, slot, fresh);
  };
  for (int c = threadIdx.x; c < p.V; c += blockDim.x) move(2 * p.G * p.D + h * p.V + c);
  if (h % per == 0)
    for (int c = threadIdx.x; c < p.D; c += blockDim.x) {
      move(grp * p.D + c);
      move((p.G + grp) * p.D + c);
    }
}

__device__ __forceinline__ void gd_copy16(float* smem, const float* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}

// Eight lanes share COLS neighbouring columns of one head's state; a lane keeps RPT key channels of each (groups of 4: 4 l ..
// 4 l + 3, then 32 further on) as packed pairs of channels. A CTA of 2 warps covers 8 COLS columns; the vectors of kGcTok
// tokens are double-buffered. Per token: two partial dots per column, a halving exchange over the eight lanes (lane bit 2 ends
// with k.S or q.S, the lower bits with the column), u by the lane that has k.S, its broadcast, the update. A lane numbers its
// columns so that the ones it hands on in the exchange always have the same registers: number c stands for column c ^ (the
// lane's column bits). Four columns a lane need the fewest instructions; with two a lone sequence's tokens follow one
// another faster. D and V multiples of 4.
constexpr int kGcThreads = 64, kGcTok = 8;

template <typename T, int RPT, int COLS>
__global__ void __launch_bounds__(kGcThreads)
gated_scan_kernel(const GatedParams p, float* __restrict__ scratch, int row0, int N) {
  constexpr int DP = 8 * RPT, P2 = RPT / 2, CTA = kGcThreads / 8 * COLS;
  constexpr int STAGE = kGcTok * (2 * DP + CTA + 4);
  static_assert(COLS == 4 || COLS == 2, "columns of a lane");
  extern __shared__ __align__(16) float gc_smem[];
  pdl_trigger();
  pdl_wait();
  const int D = p.D, V = p.V, cbs = (V + CTA - 1) / CTA;
  const int h = blockIdx.x / cbs, cb = blockIdx.x - h * cbs, j = blockIdx.y, grp = h / (p.H / p.G);
  const int t0 = p.cu[j] - row0, t1 = p.cu[j + 1] - row0, slot = p.slots[j];
  if (t1 <= t0) return;
  const GatedScratch sc = gd_scratch(scratch, N, p.H, p.G, D, V);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l8 = lane & 7;
  if (slot < 0) {
    for (int i = threadIdx.x; i < (t1 - t0) * CTA; i += kGcThreads) {
      const int c = cb * CTA + i % CTA;
      if (c < V) sc.o[(static_cast<size_t>(t0 + i / CTA) * p.H + h) * V + c] = 0.f;
    }
    return;
  }
  const bool fresh = p.reset[j] != 0;
  if (cb == 0) write_tail<T>(p, h, t0 + row0, t1 + row0, slot, fresh);
  const int flip = COLS == 4 ? l8 & 3 : (l8 >> 1) & 1;                 // the lane's column bits
  const int c_in = (threadIdx.x >> 3) * COLS, col0 = cb * CTA + c_in, own = col0 + flip;
  const bool reads_q = (l8 & 4) != 0, writes = reads_q && (COLS == 4 || (l8 & 1) == 0) && own < V;
  const auto chan = [&](int r) { return (r >> 2) * 32 + 4 * l8 + (r & 3); };
  float* S = p.memory + (static_cast<size_t>(slot) * p.H + h) * D * V;
  f32x2 s[P2][COLS];
#pragma unroll
  for (int r = 0; r < P2; ++r)
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
      const int col = col0 + (c ^ flip);
      const bool ok = chan(2 * r) < D && col < V && !fresh;            // (D is even: both channels of a pair are in or out)
      s[r][c] = ok ? pack2(S[static_cast<size_t>(chan(2 * r)) * V + col], S[static_cast<size_t>(chan(2 * r + 1)) * V + col]) : 0ull;
    }
  for (int i = threadIdx.x; i < 2 * STAGE; i += kGcThreads) gc_smem[i] = 0.f;     // channels beyond D stay zero
  __syncthreads();
  const auto load = [&](int c0, int buf) {
    float* st = gc_smem + buf * STAGE;
    const int nt = min(kGcTok, t1 - c0);
    if (4 * lane < D) {
      const size_t src = (static_cast<size_t>(c0) * p.G + grp) * D + 4 * lane;
      for (int t = warp; t < nt; t += kGcThreads / 32) {
        gd_copy16(st + t * 2 * DP + 4 * lane, sc.k + src + static_cast<size_t>(t) * p.G * D);
        gd_copy16(st + t * 2 * DP + DP + 4 * lane, sc.q + src + static_cast<size_t>(t) * p.G * D);
      }
    }
    float* vs = st + kGcTok * 2 * DP;
    constexpr int Q = CTA / 4;
    for (int i = threadIdx.x; i < nt * Q; i += kGcThreads) {
      const int t = i / Q, c = (i - t * Q) * 4;
      if (cb * CTA + c < V) gd_copy16(vs + t * CTA + c, sc.v + (static_cast<size_t>(c0 + t) * p.H + h) * V + cb * CTA + c);
    }
    float* rs = vs + kGcTok * CTA;
    if (static_cast<int>(threadIdx.x) < nt) gd_copy16(rs + threadIdx.x * 4, sc.rates + (static_cast<size_t>(c0 + threadIdx.x) * p.H + h) * 4);
  };
  load(t0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  int buf = 0;
  for (int c0 = t0; c0 < t1; c0 += kGcTok, buf ^= 1) {
    if (c0 + kGcTok < t1) load(c0 + kGcTok, buf ^ 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const float* st = gc_smem + buf * STAGE + 4 * l8;
    const float* vs = gc_smem + buf * STAGE + kGcTok * 2 * DP + c_in + flip;
    const float* rs = gc_smem + buf * STAGE + kGcTok * (2 * DP + CTA);
    float* o = sc.o + (static_cast<size_t>(c0) * p.H + h) * V + own;
    const int nt = min(kGcTok, t1 - c0);
    for (int t = 0; t < nt; ++t, st += 2 * DP, vs += CTA, rs += 4, o += static_cast<size_t>(p.H) * V) {
      f32x2 k[P2], q[P2];
#pragma unroll
      for (int r = 0; r < P2; r += 2) {
        const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(st + r * 16), b = *reinterpret_cast<const ulonglong2*>(st + DP + r * 16);
        k[r] = a.x, k[r + 1] = a.y, q[r] = b.x, q[r + 1] = b.y;
      }
      const float4 rate = *reinterpret_cast<const float4*>(rs);        // g, beta, q.k
      const float v = *vs;
      f32x2 kd[COLS], qd[COLS];
#pragma unroll
      for (int c = 0; c < COLS; ++c) kd[c] = mul2(k[0], s[0][c]), qd[c] = mul2(q[0], s[0][c]);
#pragma unroll
      for (int r = 1; r < P2; ++r)
#pragma unroll
        for (int c = 0; c < COLS; ++c) {
          kd[c] = fma2(k[r], s[r][c], kd[c]);
          qd[c] = fma2(q[r], s[r][c], qd[c]);
        }
      float x[COLS];
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        const float a = sum2(kd[c]), b = sum2(qd[c]);
        x[c] = (reads_q ? b : a) + __shfl_xor_sync(0xffffffffu, reads_q ? a : b, 4);
      }
      float y;
      if constexpr (COLS == 4) {
        const float y0 = x[0] + __shfl_xor_sync(0xffffffffu, x[2], 2), y1 = x[1] + __shfl_xor_sync(0xffffffffu, x[3], 2);
        y = y0 + __shfl_xor_sync(0xffffffffu, y1, 1);
      } else {
        y = x[0] + __shfl_xor_sync(0xffffffffu, x[1], 2);
        y += __shfl_xor_sync(0xffffffffu, y, 1);
      }
      y *= rate.x;                                                     // column `own` of the decayed state with k or q
      const float mine = rate.y * (v - y);                             // (of use where this lane has k.S)
      float u[COLS];
#pragma unroll
      for (int c = 0; c < COLS; ++c) u[c] = __shfl_sync(0xffffffffu, mine, (lane & 24) + (COLS == 4 ? c ^ flip : 2 * (c ^ flip)));
      if (writes) *o = fmaf(rate.z, u[0], y);
      const f32x2 g2 = pack2(rate.x, rate.x);
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        const f32x2 u2 = pack2(u[c], u[c]);
#pragma unroll
        for (int r = 0; r < P2; ++r) s[r][c] = fma2(k[r], u2, mul2(g2, s[r][c]));
      }
    }
    __syncthreads();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int r = 0; r < P2; ++r)
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
      const int col = col0 + (c ^ flip);
      if (chan(2 * r) >= D || col >= V) continue;
      float a, b;
      asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(s[r][c]));
      S[static_cast<size_t>(chan(2 * r)) * V + col] = a;
      S[static_cast<size_t>(chan(2 * r + 1)) * V + col] = b;
    }
}

// Any sizes: one CTA per (head, piece), a thread owns state columns, the state stays in global memory.
template <typename T>
__global__ void __launch_bounds__(256)
gated_scan_any_kernel(const GatedParams p, float* __restrict__ scratch, int row0, int N) {
  pdl_trigger();
  pdl_wait();
  const int D = p.D, V = p.V, h = blockIdx.x, j = blockIdx.y, grp = h / (p.H / p.G);
  const int t0 = p.cu[j] - row0, t1 = p.cu[j + 1] - row0, slot = p.slots[j];
  if (t1 <= t0) return;
  const GatedScratch sc = gd_scratch(scratch, N, p.H, p.G, D, V);
  const bool fresh = p.reset[j] != 0;
  if (slot >= 0) write_tail<T>(p, h, t0 + row0, t1 + row0, slot, fresh);
  float* S = p.memory + (static_cast<size_t>(max(slot, 0)) * p.H + h) * D * V;
  for (int c = threadIdx.x; c < V; c += blockDim.x) {
    for (int i = 0; fresh && slot >= 0 && i < D; ++i) S[static_cast<size_t>(i) * V + c] = 0.f;
    for (int t = t0; t < t1; ++t) {
      float* o = sc.o + (static_cast<size_t>(t) * p.H + h) * V + c;
      if (slot < 0) {
        *o = 0.f;
        continue;
      }
      const float* k = sc.k + (static_cast<size_t>(t) * p.G + grp) * D;
      const float* q = sc.q + (static_cast<size_t>(t) * p.G + grp) * D;
      const float* r = sc.rates + (static_cast<size_t>(t) * p.H + h) * 4;
      float kk = 0.f, qq = 0.f;
      for (int i = 0; i < D; ++i) {
        const float s = S[static_cast<size_t>(i) * V + c];
        kk = fmaf(k[i], s, kk);
        qq = fmaf(q[i], s, qq);
      }
      const float g = r[0], u = r[1] * (sc.v[(static_cast<size_t>(t) * p.H + h) * V + c] - g * kk);
      for (int i = 0; i < D; ++i) {
        float* s = S + static_cast<size_t>(i) * V + c;
        *s = fmaf(k[i], u, g * *s);
      }
      *o = fmaf(g, qq, r[2] * u);
    }
  }
}

// One warp per (token, head): o / rms(o) * norm_w * silu(gate).
template <typename T>
__global__ void __launch_bounds__(256)
gated_post_kernel(const GatedParams p, float* __restrict__ scratch, int row0, int N) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, V = p.V;
  const unsigned gw = blockIdx.x * (blockDim.x / 32) + (threadIdx.x >> 5);
  if (gw >= static_cast<unsigned>(N) * p.H) return;
  const int n = static_cast<int>(gw / p.H), h = static_cast<int>(gw - static_cast<unsigned>(n) * p.H);
  const GatedScratch sc = gd_scratch(scratch, N, p.H, p.G, p.D, V);
  const float* o = sc.o + (static_cast<size_t>(n) * p.H + h) * V;
  const T* z = static_cast<const T*>(p.proj) + static_cast<size_t>(row0 + n) * p.ld + gd_channels(p) + h * V;
  T* out = static_cast<T*>(p.out) + (static_cast<size_t>(row0 + n) * p.H + h) * V;
  const bool vec = V % 4 == 0 && p.D % 2 == 0 && p.ld % 4 == 0 && gd_channels(p) % 4 == 0;    // every group aligned
  float s = 0.f;
  if (vec) {
    for (int c = 4 * lane; c < V; c += 128) {
      float a[4];
      load_v<4>(o + c, a);
#pragma unroll
      for (int e = 0; e < 4; ++e) s = fmaf(a[e], a[e], s);
    }
    const float rs = 1.f / sqrtf(warp_sum(s) / V + p.norm_eps);
    for (int c = 4 * lane; c < V; c += 128) {
      float a[4], g[4];
      load_v<4>(o + c, a);
      load_v<4>(z + c, g);
#pragma unroll
      for (int e = 0; e < 4; ++e) a[e] *= rs * p.norm_w[c + e] * silu_f(g[e]);
      store_v<4>(out + c, a);
    }
    return;
  }
  for (int c = lane; c < V; c += 32) s = fmaf(o[c], o[c], s);
  const float rs = 1.f / sqrtf(warp_sum(s) / V + p.norm_eps);
  for (int c = lane; c < V; c += 32) out[c] = from_f<T>(o[c] * rs * p.norm_w[c] * silu_f(to_f(z[c])));
}

template <typename T>
static int launch_gated_step(const GatedParams& p, int pieces, cudaStream_t st) {
  const dim3 grid(p.G, pieces), block(kGsThreads);
  const size_t smem = static_cast<size_t>(p.H / p.G) * p.V * sizeof(float);
  if (p.D <= 32) return static_cast<int>(launch_kernel(gated_step_kernel<T, 4>, grid, block, smem, st, p));
  if (p.D <= 64) return static_cast<int>(launch_kernel(gated_step_kernel<T, 8>, grid, block, smem, st, p));
  return static_cast<int>(launch_kernel(gated_step_kernel<T, 16>, grid, block, smem, st, p));
}

template <typename T, int RPT, int COLS>
static int launch_gated_scan_cols(const GatedParams& p, float* scratch, int pieces, int row0, int N, cudaStream_t st) {
  constexpr int CTA = kGcThreads / 8 * COLS, smem = 2 * kGcTok * (2 * 8 * RPT + CTA + 4) * 4;
  static_assert(smem <= 48 * 1024, "fits the default limit");
  const int cbs = (p.V + CTA - 1) / CTA;
  return static_cast<int>(launch_kernel(gated_scan_kernel<T, RPT, COLS>, dim3(p.H * cbs, pieces), dim3(kGcThreads), smem, st, p, scratch, row0, N));
}

template <typename T, int RPT>
static int launch_gated_scan(const GatedParams& p, float* scratch, int pieces, int row0, int N, cudaStream_t st) {
  // columns of a lane: two while that leaves every SM no more than one CTA
  const bool few = static_cast<long long>(pieces) * p.H * ((p.V + 15) / 16) <= 148;
  return few ? launch_gated_scan_cols<T, RPT, 2>(p, scratch, pieces, row0, N, st) : launch_gated_scan_cols<T, RPT, 4>(p, scratch, pieces, row0, N, st);
}

static bool gated_step_covered(int H, int G, int D, int V) {
  return D <= 128 && V <= 128 && V % 4 == 0 && static_cast<long long>(H / G) * V * 4 <= 32 * 1024;
}

template <typename T>
static int gated_delta_typed(GatedParams p, int pieces, int n_short, int rows, float* scratch, int mode, cudaStream_t st) {
  const size_t ab = sizeof(T) * 4;
  const bool vec = p.D % 4 == 0 && p.V % 4 == 0 && p.ld % 4 == 0 && aligned_to(p.proj, ab) && aligned_to(p.out, ab) &&
                   aligned_to(scratch, 16) && aligned_to(p.memory, 16);
  if (n_short > 0) {
    if (!gated_step_covered(p.H, p.G, p.D, p.V) || !aligned_to(p.memory, 16)) return -1;
    const int rc = launch_gated_step<T>(p, n_short, st);
    if (rc) return rc;
  }
  const int np = pieces - n_short, N = rows - n_short;
  if (np <= 0 || N <= 0) return 0;
  if (scratch == nullptr) return -1;
  p.slots += n_short, p.cu += n_short, p.reset += n_short, p.pieces = np;
  const bool fast = mode == 0 && vec && p.D <= 128 && p.V <= 128;
  int rc;
  const unsigned units = p.G + p.H;
  const dim3 run((N + kGpTok * (kGpThreads / 32) - 1) / (kGpTok * (kGpThreads / 32)), units), one((N + kGpThreads / 32 - 1) / (kGpThreads / 32), units);
  if (fast && p.taps == 4) rc = static_cast<int>(launch_kernel(gated_prep_kernel<T, 4>, run, dim3(kGpThreads), 0, st, p, scratch, n_short, N));
  else if (fast && p.taps == 3) rc = static_cast<int>(launch_kernel(gated_prep_kernel<T, 3>, run, dim3(kGpThreads), 0, st, p, scratch, n_short, N));
  else if (fast && p.taps == 2) rc = static_cast<int>(launch_kernel(gated_prep_kernel<T, 2>, run, dim3(kGpThreads), 0, st, p, scratch, n_short, N));
  else rc = static_cast<int>(launch_kernel(gated_prep_any_kernel<T>, one, dim3(kGpThreads), 0, st, p, scratch, n_short, N));
  if (rc) return rc;
  if (!fast) rc = static_cast<int>(launch_kernel(gated_scan_any_kernel<T>, dim3(p.H, np), dim3(p.V <= 128 ? 128 : 256), 0, st, p, scratch, n_short, N));
  else if (p.D <= 32) rc = launch_gated_scan<T, 4>(p, scratch, np, n_short, N, st);
  else if (p.D <= 64) rc = launch_gated_scan<T, 8>(p, scratch, np, n_short, N, st);
  else rc = launch_gated_scan<T, 16>(p, scratch, np, n_short, N, st);
  if (rc) return rc;
  const long long warps = static_cast<long long>(N) * p.H;
  if (warps > 0x7fffffffll) return -1;
  return static_cast<int>(launch_kernel(gated_post_kernel<T>, dim3(static_cast<unsigned>((warps + 7) / 8)), dim3(256), 0, st, p, scratch, n_short, N));
}

}  // namespace mx

using namespace mx;

extern "C" long long mx_gated_delta_scratch_floats(int tokens, int H, int G, int D, int V) {
  return static_cast<long long>(tokens) * (4ll * H + 2ll * G * D + 2ll * H * V);
}

// Whether one-token pieces of these sizes have a kernel of their own (else they count as longer pieces).
extern "C" int mx_gated_delta_step_covered(int H, int G, int D, int V, int taps) { return taps >= 1 && gated_step_covered(H, G, D, V) ? 1 : 0; }

// A ragged batch of pieces (token rows cu[j] .. cu[j + 1] - 1 of proj, rates and out, state slot slots[j], reset[j] starts
// from zero). The first n_short pieces hold exactly one token each (and need mx_gated_delta_step_covered); rows is the
// total number of token rows. scratch: mx_gated_delta_scratch_floats(rows - n_short, ...) floats, or NULL when every piece
// is short. mode 1 forces the kernels that cover any size.
extern "C" int mx_gated_delta(const void* proj, long long ld, const void* rates, const void* conv_w, const void* A_log,
                              const void* dt_bias, const void* norm_w, void* memory, void* tail, const void* slots, const void* cu,
                              const void* reset, void* out, void* scratch, int pieces, int n_short, int rows, int H, int G, int D, int V,
                              int taps, float unit_eps, float norm_eps, int fp32, int mode, void* stream) {
  if (pieces <= 0 || rows <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || taps <= 0 || pieces > 65535 || G + H > 65535 || n_short < 0 || n_short > pieces) return -1;
  GatedParams p{proj, ld, static_cast<const float*>(rates), static_cast<const float*>(conv_w), static_cast<const float*>(A_log),
                static_cast<const float*>(dt_bias), static_cast<const float*>(norm_w), static_cast<float*>(memory), static_cast<float*>(tail),
                static_cast<const int*>(slots), static_cast<const int*>(cu), static_cast<const int*>(reset), out, H, G, D, V, taps, pieces,
                unit_eps, norm_eps};
  auto st = static_cast<cudaStream_t>(stream);
  auto* sc = static_cast<float*>(scratch);
  return fp32 ? gated_delta_typed<float>(p, pieces, n_short, rows, sc, mode, st)
              : gated_delta_typed<__nv_bfloat16>(p, pieces, n_short, rows, sc, mode, st);
}
