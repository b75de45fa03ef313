// Generalized delta rule with a decay and a removal rate per head and key channel:
//   u = k / sqrt(|k|^2 + unit_eps),  w = exp(-decay_scale * sigmoid(w0 + W2 tanh(l))),  a = sigmoid(a_in + a_bias)
//   S <- diag(w) S - (a u)(u^T S) + k v^T      (both terms read the old state)
//   o  = S^T r,  out = o / rms(o) * norm_w * sigmoid(g)
// State [slots, H, D, D] fp32 (key channel major). Everything that enters the recurrence is fp32.
//
// Writing p = u^T S_old and n = sqrt(|k|^2 + unit_eps), the output needs the old state only:
//   o = (r w)^T S_old - (sum r a u) p + n (sum r u) v,   S_ij <- w_i S_ij + u_i (n v_j - a_i p_j)
// so a step is one pass of two dot products per state column, one reduction round and one update.
//
// Kernels:
//   delta_any    any sizes, any piece length: one CTA per (head, piece), state in global memory
//   delta_step   pieces of one token (decode): one CTA per (head, row), the state passes through
//                registers once, preparation and output norm fused
//   delta_prep / delta_scan / delta_post   longer pieces: the per-token vectors for all tokens at once,
//                the recurrence with the state in registers, the per-head norm and gate
#include "api.h"
#include "typed.cuh"

namespace mx {

struct DeltaParams {
  const void* proj;          // rows r | k | v | g | a | l at stride ld, offsets below
  long long ld;
  int off_r, off_k, off_v, off_g, off_a, off_l;
  const void* w2;            // [H * D, R], activation type
  const float* w0;           // [H * D]
  const float* a_bias;       // [H * D]
  const float* norm_w;       // [H * D]
  float* state;
  const int* slots;          // per piece; a negative slot marks a padding row (its output is zero)
  const int* cu;
  const int* reset;
  void* out;                 // [rows, H * D]
  int H, D, R;
  float decay_scale, unit_eps, norm_eps;
};

// Decay of one channel from its low-rank pre-activation. Slow channels sit just below one and are multiplied
// into the state at every token, so an error of the exponential there grows with the distance: 1 + expm1
// is within half a unit in the last place of the exact value, expf within two.
__device__ __forceinline__ float channel_decay(float z, float scale) { return 1.f + expm1f(-scale * sigmoid_f(z)); }

template <typename T>
__device__ __forceinline__ float low_rank_dot(const T* __restrict__ w2_row, const float* __restrict__ tl, int R, bool vec) {
  float z = 0.f;
  if (vec) {
    for (int i = 0; i < R; i += 4) {
      float f[4];
      load_v<4>(w2_row + i, f);
      z = fmaf(f[0], tl[i], z);
      z = fmaf(f[1], tl[i + 1], z);
      z = fmaf(f[2], tl[i + 2], z);
      z = fmaf(f[3], tl[i + 3], z);
    }
  } else {
    for (int i = 0; i < R; ++i) z = fmaf(to_f(w2_row[i]), tl[i], z);
  }
  return z;
}

// ----------------------------------------------------------------------------- any sizes
template <typename T>
__global__ void __launch_bounds__(256) delta_any_kernel(const DeltaParams p) {
  extern __shared__ float dg_smem[];
  __shared__ float red[3 * 33];
  const int D = p.D, R = p.R;
  float* tl = dg_smem;          // [R rounded up to 4]
  float* u_s = tl + ((R + 3) & ~3);
  float* a_s = u_s + D;
  float* w_s = a_s + D;
  float* rw_s = w_s + D;
  float* o_s = rw_s + D;
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, j = blockIdx.y;
  const int t0 = p.cu[j], t1 = p.cu[j + 1], slot = p.slots[j];
  T* out = static_cast<T*>(p.out);
  const int hd = h * D, HD = p.H * D;
  if (slot < 0) {
    for (int t = t0; t < t1; ++t)
      for (int i = threadIdx.x; i < D; i += blockDim.x) out[static_cast<size_t>(t) * HD + hd + i] = from_f<T>(0.f);
    return;
  }
  float* S = p.state + (static_cast<size_t>(slot) * p.H + h) * D * D;
  if (p.reset[j])
    for (int c = threadIdx.x; c < D; c += blockDim.x)
      for (int i = 0; i < D; ++i) S[static_cast<size_t>(i) * D + c] = 0.f;     // (a thread owns its columns)
  for (int t = t0; t < t1; ++t) {
    const T* row = static_cast<const T*>(p.proj) + static_cast<size_t>(t) * p.ld;
    __syncthreads();
    for (int i = threadIdx.x; i < R; i += blockDim.x) tl[i] = tanhf(to_f(row[p.off_l + i]));
    float s[3] = {0.f, 0.f, 0.f};
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
      const float k = to_f(row[p.off_k + hd + i]);
      s[0] += k * k;
    }
    block_sums<3>(s, red);
    const float n = sqrtf(s[0] + p.unit_eps), inv = 1.f / n;
    s[0] = s[1] = s[2] = 0.f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
      const float z = p.w0[hd + i] + low_rank_dot(static_cast<const T*>(p.w2) + static_cast<size_t>(hd + i) * R, tl, R, false);
      const float w = channel_decay(z, p.decay_scale), a = sigmoid_f(to_f(row[p.off_a + hd + i]) + p.a_bias[hd + i]);
      const float u = to_f(row[p.off_k + hd + i]) * inv, r = to_f(row[p.off_r + hd + i]);
      u_s[i] = u, a_s[i] = a, w_s[i] = w, rw_s[i] = r * w;
      s[0] += r * a * u;
      s[1] += r * u;
    }
    block_sums<3>(s, red);
    const float rau = s[0], ru = s[1];
    float ssq[1] = {0.f};
    for (int c = threadIdx.x; c < D; c += blockDim.x) {
      float pr = 0.f, oo = 0.f;
      for (int i = 0; i < D; ++i) {
        const float v = S[static_cast<size_t>(i) * D + c];
        pr = fmaf(u_s[i], v, pr);
        oo = fmaf(rw_s[i], v, oo);
      }
      const float nv = n * to_f(row[p.off_v + hd + c]);
      for (int i = 0; i < D; ++i) {
        float* e = S + static_cast<size_t>(i) * D + c;
        *e = fmaf(w_s[i], *e, u_s[i] * fmaf(-a_s[i], pr, nv));
      }
      const float o = oo - rau * pr + ru * nv;
      o_s[c] = o;
      ssq[0] += o * o;
    }
    block_sums<1>(ssq, red);
    const float rs = 1.f / sqrtf(ssq[0] / D + p.norm_eps);
    for (int c = threadIdx.x; c < D; c += blockDim.x)
      out[static_cast<size_t>(t) * HD + hd + c] =
          from_f<T>(o_s[c] * rs * p.norm_w[hd + c] * sigmoid_f(to_f(row[p.off_g + hd + c])));
  }
}

// ----------------------------------------------------------------------------- one token per piece
// 8 warps; warp q holds state rows q, q + 8, ... (RPW of them) and lane c the columns 4c .. 4c + 3, so the
// state is read and written once in 16-byte pieces (D % 4 == 0, D <= 128).
template <typename T, int RPW>
__global__ void __launch_bounds__(256) delta_step_kernel(const DeltaParams p) {
  extern __shared__ __align__(16) float ds_tl[];            // [R rounded up to 4]
  __shared__ float red[3 * 33];
  __shared__ float u_s[128], a_s[128], w_s[128], rw_s[128];
  __shared__ __align__(16) float pr_s[128];
  __shared__ __align__(16) float part[8][2][128];
  pdl_trigger();
  pdl_wait();
  const int D = p.D, R = p.R, h = blockIdx.x, j = blockIdx.y;
  const int hd = h * D, HD = p.H * D;
  const int t = p.cu[j], slot = p.slots[j], tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(t) * HD + hd;
  if (slot < 0) {
    if (tid < D) out[tid] = from_f<T>(0.f);
    return;
  }
  float* S = p.state + (static_cast<size_t>(slot) * p.H + h) * D * D;
  const bool fresh = p.reset[j] != 0, col_ok = 4 * lane < D;
  float4 st[RPW];
#pragma unroll
  for (int q = 0; q < RPW; ++q) {
    const int i = warp + 8 * q;
    st[q] = (col_ok && i < D && !fresh) ? *reinterpret_cast<const float4*>(S + static_cast<size_t>(i) * D + 4 * lane)
                                        : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const T* row = static_cast<const T*>(p.proj) + static_cast<size_t>(t) * p.ld;
  for (int i = tid; i < R; i += 256) ds_tl[i] = tanhf(to_f(row[p.off_l + i]));
  const bool ch = tid < D;
  const float k = ch ? to_f(row[p.off_k + hd + tid]) : 0.f, r = ch ? to_f(row[p.off_r + hd + tid]) : 0.f;
  float s[3] = {k * k, 0.f, 0.f};
  block_sums<3>(s, red);                      // (also publishes tanh(l))
  const float n = sqrtf(s[0] + p.unit_eps);
  s[0] = s[1] = s[2] = 0.f;
  if (ch) {
    const T* w2 = static_cast<const T*>(p.w2) + static_cast<size_t>(hd + tid) * R;
    const float z = p.w0[hd + tid] + low_rank_dot(w2, ds_tl, R, R % 4 == 0);
    const float w = channel_decay(z, p.decay_scale), a = sigmoid_f(to_f(row[p.off_a + hd + tid]) + p.a_bias[hd + tid]);
    const float u = k / n;
    u_s[tid] = u, a_s[tid] = a, w_s[tid] = w, rw_s[tid] = r * w;
    s[0] = r * a * u;
    s[1] = r * u;
  }
  block_sums<3>(s, red);
  const float rau = s[0], ru = s[1];
  float4 pr = make_float4(0.f, 0.f, 0.f, 0.f), oo = pr;
#pragma unroll
  for (int q = 0; q < RPW; ++q) {
    const int i = warp + 8 * q;
    if (i < D) {
      const float u = u_s[i], rw = rw_s[i];
      pr.x = fmaf(u, st[q].x, pr.x), pr.y = fmaf(u, st[q].y, pr.y), pr.z = fmaf(u, st[q].z, pr.z), pr.w = fmaf(u, st[q].w, pr.w);
      oo.x = fmaf(rw, st[q].x, oo.x), oo.y = fmaf(rw, st[q].y, oo.y), oo.z = fmaf(rw, st[q].z, oo.z), oo.w = fmaf(rw, st[q].w, oo.w);
    }
  }
  *reinterpret_cast<float4*>(&part[warp][0][4 * lane]) = pr;
  *reinterpret_cast<float4*>(&part[warp][1][4 * lane]) = oo;
  __syncthreads();
  float o = 0.f;
  if (ch) {
    float prj = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) prj += part[w][0][tid], o += part[w][1][tid];
    const float nv = n * to_f(row[p.off_v + hd + tid]);
    o = o - rau * prj + ru * nv;
    pr_s[tid] = prj;
    part[0][0][tid] = nv;                     // (this thread has read its column of every warp's partial)
  }
  s[0] = o * o, s[1] = s[2] = 0.f;
  block_sums<3>(s, red);                      // (also publishes pr_s and n v)
  if (ch) {
    const float rs = 1.f / sqrtf(s[0] / D + p.norm_eps);
    out[tid] = from_f<T>(o * rs * p.norm_w[hd + tid] * sigmoid_f(to_f(row[p.off_g + hd + tid])));
  }
  if (!col_ok) return;
  const float4 pv = *reinterpret_cast<const float4*>(&pr_s[4 * lane]);
  const float4 nv = *reinterpret_cast<const float4*>(&part[0][0][4 * lane]);
#pragma unroll
  for (int q = 0; q < RPW; ++q) {
    const int i = warp + 8 * q;
    if (i < D) {
      const float u = u_s[i], a = -a_s[i], w = w_s[i];
      float4 v;
      v.x = fmaf(w, st[q].x, u * fmaf(a, pv.x, nv.x));
      v.y = fmaf(w, st[q].y, u * fmaf(a, pv.y, nv.y));
      v.z = fmaf(w, st[q].z, u * fmaf(a, pv.z, nv.z));
      v.w = fmaf(w, st[q].w, u * fmaf(a, pv.w, nv.w));
      *reinterpret_cast<float4*>(S + static_cast<size_t>(i) * D + 4 * lane) = v;
    }
  }
}

// ----------------------------------------------------------------------------- longer pieces
// Scratch of one call over N tokens (token rows row0 .. row0 + N - 1), fp32:
//   five arrays [N, H * D]: w, a, u, r w, n v;  two arrays [N, H]: sum r a u, sum r u;  o [N, H * D]
constexpr int kPrepTok = 16;

template <typename T>
__global__ void __launch_bounds__(256)
delta_prep_kernel(const DeltaParams p, float* __restrict__ scratch, int row0, int N) {
  extern __shared__ __align__(16) float dp_smem[];
  const int D = p.D, R = p.R, Rp = (R + 3) & ~3, h = blockIdx.y, hd = h * D;
  const size_t HD = static_cast<size_t>(p.H) * D;
  float* tl = dp_smem;                        // [kPrepTok][Rp]
  float* zs = tl + kPrepTok * Rp;             // [kPrepTok][D]
  pdl_trigger();
  pdl_wait();
  const int n0 = blockIdx.x * kPrepTok, nt = min(kPrepTok, N - n0);
  const T* base = static_cast<const T*>(p.proj) + static_cast<size_t>(row0 + n0) * p.ld;
  for (int i = threadIdx.x; i < kPrepTok * Rp; i += 256) {
    const int t = i / Rp, c = i - t * Rp;
    tl[i] = (t < nt && c < R) ? tanhf(to_f(base[static_cast<size_t>(t) * p.ld + p.off_l + c])) : 0.f;
  }
  __syncthreads();
  // low-rank product: a thread owns one channel for half of the tokens
  constexpr int TH = kPrepTok / 2;
  const int half = threadIdx.x >> 7;
  for (int i = threadIdx.x & 127; i < D; i += 128) {
    float acc[TH];
    const float z0 = p.w0[hd + i];
#pragma unroll
    for (int t = 0; t < TH; ++t) acc[t] = 0.f;
    const T* w2 = static_cast<const T*>(p.w2) + static_cast<size_t>(hd + i) * R;
    const float* tb = tl + half * TH * Rp;
    if (R % 4 == 0) {
      for (int c = 0; c < R; c += 4) {
        float f[4];
        load_v<4>(w2 + c, f);
#pragma unroll
        for (int t = 0; t < TH; ++t) {
          const float4 x = *reinterpret_cast<const float4*>(tb + t * Rp + c);
          acc[t] = fmaf(f[0], x.x, acc[t]);
          acc[t] = fmaf(f[1], x.y, acc[t]);
          acc[t] = fmaf(f[2], x.z, acc[t]);
          acc[t] = fmaf(f[3], x.w, acc[t]);
        }
      }
    } else {
      for (int c = 0; c < R; ++c) {
        const float f = to_f(w2[c]);
#pragma unroll
        for (int t = 0; t < TH; ++t) acc[t] = fmaf(f, tb[t * Rp + c], acc[t]);
      }
    }
#pragma unroll
    for (int t = 0; t < TH; ++t) zs[(half * TH + t) * D + i] = z0 + acc[t];
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t arr = static_cast<size_t>(N) * HD;
  float* sums = scratch + 5 * arr;
  for (int t = warp; t < nt; t += 8) {
    const T* row = base + static_cast<size_t>(t) * p.ld;
    float kk = 0.f;
    for (int i = lane; i < D; i += 32) {
      const float k = to_f(row[p.off_k + hd + i]);
      kk += k * k;
    }
    const float n = sqrtf(warp_sum(kk) + p.unit_eps), inv = 1.f / n;
    float rau = 0.f, ru = 0.f;
    float* dst = scratch + static_cast<size_t>(n0 + t) * HD + hd;
    for (int i = lane; i < D; i += 32) {
      const float w = channel_decay(zs[t * D + i], p.decay_scale);
      const float a = sigmoid_f(to_f(row[p.off_a + hd + i]) + p.a_bias[hd + i]);
      const float u = to_f(row[p.off_k + hd + i]) * inv, r = to_f(row[p.off_r + hd + i]);
      dst[i] = w;
      dst[arr + i] = a;
      dst[2 * arr + i] = u;
      dst[3 * arr + i] = r * w;
      dst[4 * arr + i] = n * to_f(row[p.off_v + hd + i]);
      rau += r * a * u;
      ru += r * u;
    }
    rau = warp_sum(rau);
    ru = warp_sum(ru);
    if (lane == 0) {
      sums[static_cast<size_t>(n0 + t) * p.H + h] = rau;
      sums[static_cast<size_t>(N) * p.H + static_cast<size_t>(n0 + t) * p.H + h] = ru;
    }
  }
}

__device__ __forceinline__ void cp_async16_g(float* smem, const float* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}
__device__ __forceinline__ void cp_async4_g(float* smem, const float* g) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}

// Half a warp (16 lanes) shares kScanCols neighbouring columns of one head's state; a lane keeps RPT
// key channels of each (channel groups of 4: 4 l .. 4 l + 3, then 64 further on; RPT = 2: 2 l, 2 l + 1), so
// that every vector element read from shared memory feeds kScanCols columns (the kernel is bound by those
// reads and by instruction issue). A CTA of 4 warps covers kScanCta columns; the vectors of kScanTok tokens
// are double-buffered. Per token: two partial dots per column, one halving exchange over the 16 lanes (lane
// bit 3 ends with p or with the state part of o, bits 2 and 1 with the column), the update.
constexpr int kScanCols = 4;
constexpr int kScanCtaThreads = 128;
constexpr int kScanCta = kScanCtaThreads / 16 * kScanCols;
constexpr int kScanTok = 8;

template <int RPT>
__global__ void __launch_bounds__(kScanCtaThreads)
delta_scan_kernel(const DeltaParams p, float* __restrict__ scratch, const int* __restrict__ slots,
                  const int* __restrict__ cu, const int* __restrict__ reset, int row0, int N) {
  constexpr int DP = 16 * RPT;
  constexpr int STAGE = kScanTok * (4 * DP + kScanCta + 2);
  extern __shared__ __align__(16) float sc_smem[];
  pdl_trigger();
  pdl_wait();
  const int D = p.D, cbs = (D + kScanCta - 1) / kScanCta;
  const int h = blockIdx.x / cbs, cb = blockIdx.x - h * cbs, j = blockIdx.y;
  const int t0 = cu[j] - row0, t1 = cu[j + 1] - row0, slot = slots[j];
  if (t1 <= t0 || slot < 0) return;
  const size_t HD = static_cast<size_t>(p.H) * D, arr = static_cast<size_t>(N) * HD;
  const int lane = threadIdx.x & 31, l16 = lane & 15, grp = threadIdx.x >> 4;
  const int c_in = grp * kScanCols, col0 = cb * kScanCta + c_in;
  const int o_col = col0 + ((l16 & 4) >> 1) + ((l16 & 2) >> 1);      // output column of this lane
  // channel of this lane's row q
  const auto chan = [&](int q) { return RPT == 2 ? 2 * l16 + q : (q >> 2) * 64 + 4 * l16 + (q & 3); };
  float* S = p.state + (static_cast<size_t>(slot) * p.H + h) * D * D;
  float s[RPT][kScanCols];
  const bool fresh = reset[j] != 0;
#pragma unroll
  for (int q = 0; q < RPT; ++q)
#pragma unroll
    for (int c = 0; c < kScanCols; ++c)
      s[q][c] = (chan(q) < D && col0 + c < D && !fresh) ? S[static_cast<size_t>(chan(q)) * D + col0 + c] : 0.f;
  // channels beyond D stay zero in both stages
  for (int i = threadIdx.x; i < 2 * STAGE; i += kScanCtaThreads) sc_smem[i] = 0.f;
  __syncthreads();
  const float* sums = scratch + 5 * arr;
  float* o_out = scratch + 5 * arr + 2 * static_cast<size_t>(N) * p.H;
  const auto load = [&](int c0, int buf) {
    float* st = sc_smem + buf * STAGE;
    const int nt = min(kScanTok, t1 - c0);
    if (nt > 0) {
      const size_t g0 = static_cast<size_t>(c0) * HD + static_cast<size_t>(h) * D;
      // one warp per array: a lane copies its four channels of every token
      const int a = threadIdx.x >> 5;
      const float* src = scratch + a * arr + g0;
      float* dst = st + a * DP;
      if (D % 4 == 0) {
        const int c = lane * 4;
        if (c < D)
          for (int t = 0; t < nt; ++t) cp_async16_g(dst + t * 4 * DP + c, src + t * HD + c);
      } else {
        for (int t = 0; t < nt; ++t)
          for (int c = lane; c < D; c += 32) cp_async4_g(dst + t * 4 * DP + c, src + t * HD + c);
      }
      float* vs = st + kScanTok * 4 * DP;
      {
        const int c = threadIdx.x % kScanCta, col = cb * kScanCta + c;
        if (col < D)
          for (int t = threadIdx.x / kScanCta; t < nt; t += kScanCtaThreads / kScanCta)
            cp_async4_g(vs + t * kScanCta + c, scratch + 4 * arr + g0 + t * HD + col);
      }
      float* ss = vs + kScanTok * kScanCta;
      for (int i = threadIdx.x; i < nt * 2; i += kScanCtaThreads)
        cp_async4_g(ss + i, sums + static_cast<size_t>(i & 1) * N * p.H + static_cast<size_t>(c0 + (i >> 1)) * p.H + h);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(t0, 0);
  int buf = 0;
  for (int c0 = t0; c0 < t1; c0 += kScanTok, buf ^= 1) {
    load(c0 + kScanTok, buf ^ 1);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const float* st = sc_smem + buf * STAGE;
    const float* vs = st + kScanTok * 4 * DP;
    const float* ss = vs + kScanTok * kScanCta;
    const int nt = min(kScanTok, t1 - c0);
    for (int t = 0; t < nt; ++t) {
      float w[RPT], a[RPT], u[RPT], rw[RPT];
      const float* v4 = st + t * 4 * DP;
      const auto fetch = [&](const float* src, float(&dst)[RPT]) {
        if constexpr (RPT == 2) {
          const float2 x = *reinterpret_cast<const float2*>(src + 2 * l16);
          dst[0] = x.x, dst[1] = x.y;
        } else {
#pragma unroll
          for (int q = 0; q < RPT; q += 4) {
            const float4 x = *reinterpret_cast<const float4*>(src + q * 16 + 4 * l16);
            dst[q] = x.x, dst[q + 1] = x.y, dst[q + 2] = x.z, dst[q + 3] = x.w;
          }
        }
      };
      fetch(v4 + 2 * DP, u);
      fetch(v4 + 3 * DP, rw);
      float pd[kScanCols], od[kScanCols];
#pragma unroll
      for (int c = 0; c < kScanCols; ++c) pd[c] = od[c] = 0.f;
#pragma unroll
      for (int q = 0; q < RPT; ++q)
#pragma unroll
        for (int c = 0; c < kScanCols; ++c) {
          pd[c] = fmaf(u[q], s[q][c], pd[c]);
          od[c] = fmaf(rw[q], s[q][c], od[c]);
        }
      fetch(v4, w);
      fetch(v4 + DP, a);
      const bool up8 = (l16 & 8) != 0, up4 = (l16 & 4) != 0, up2 = (l16 & 2) != 0;
      float x[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) x[c] = (up8 ? od[c] : pd[c]) + __shfl_xor_sync(0xffffffffu, up8 ? pd[c] : od[c], 8);
      const float y0 = (up4 ? x[2] : x[0]) + __shfl_xor_sync(0xffffffffu, up4 ? x[0] : x[2], 4);
      const float y1 = (up4 ? x[3] : x[1]) + __shfl_xor_sync(0xffffffffu, up4 ? x[1] : x[3], 4);
      float y = (up2 ? y1 : y0) + __shfl_xor_sync(0xffffffffu, up2 ? y0 : y1, 2);
      y += __shfl_xor_sync(0xffffffffu, y, 1);
      float pc[kScanCols];
#pragma unroll
      for (int c = 0; c < kScanCols; ++c) pc[c] = __shfl_sync(0xffffffffu, y, (lane & 16) + 2 * c);
      const float4 nv4 = *reinterpret_cast<const float4*>(vs + t * kScanCta + c_in);
      const float nv[kScanCols] = {nv4.x, nv4.y, nv4.z, nv4.w};
      if (up8 && (l16 & 1) == 0 && o_col < D) {
        const float pp = up4 ? (up2 ? pc[3] : pc[2]) : (up2 ? pc[1] : pc[0]);
        const float vv = up4 ? (up2 ? nv[3] : nv[2]) : (up2 ? nv[1] : nv[0]);
        o_out[static_cast<size_t>(c0 + t) * HD + h * D + o_col] = y - ss[2 * t] * pp + ss[2 * t + 1] * vv;
      }
#pragma unroll
      for (int q = 0; q < RPT; ++q)
#pragma unroll
        for (int c = 0; c < kScanCols; ++c) s[q][c] = fmaf(w[q], s[q][c], u[q] * fmaf(-a[q], pc[c], nv[c]));
    }
    __syncthreads();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int q = 0; q < RPT; ++q)
#pragma unroll
    for (int c = 0; c < kScanCols; ++c)
      if (chan(q) < D && col0 + c < D) S[static_cast<size_t>(chan(q)) * D + col0 + c] = s[q][c];
}

// One warp per (token, head): o / rms(o) * norm_w * sigmoid(g).
template <typename T>
__global__ void __launch_bounds__(256)
delta_post_kernel(const DeltaParams p, const float* __restrict__ scratch, int row0, int N) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, D = p.D;
  const long long gw = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) >> 5;
  if (gw >= static_cast<long long>(N) * p.H) return;
  const int t = static_cast<int>(gw / p.H), h = static_cast<int>(gw - static_cast<long long>(t) * p.H), hd = h * D;
  const size_t HD = static_cast<size_t>(p.H) * D;
  const float* o = scratch + 5 * static_cast<size_t>(N) * HD + 2 * static_cast<size_t>(N) * p.H + static_cast<size_t>(t) * HD + hd;
  const T* g = static_cast<const T*>(p.proj) + static_cast<size_t>(row0 + t) * p.ld + p.off_g + hd;
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(row0 + t) * HD + hd;
  float s = 0.f;
  for (int i = lane; i < D; i += 32) s += o[i] * o[i];
  const float rs = 1.f / sqrtf(warp_sum(s) / D + p.norm_eps);
  for (int i = lane; i < D; i += 32) out[i] = from_f<T>(o[i] * rs * p.norm_w[hd + i] * sigmoid_f(to_f(g[i])));
}

template <typename T>
static int launch_delta_any(const DeltaParams& p, int pieces, cudaStream_t st) {
  const size_t smem = (5 * static_cast<size_t>(p.D) + ((p.R + 3) & ~3)) * sizeof(float);
  if (smem > 40 * 1024) return -1;
  return static_cast<int>(launch_kernel(delta_any_kernel<T>, dim3(p.H, pieces), dim3(256), smem, st, p));
}

template <typename T>
static int launch_delta_step(const DeltaParams& p, int pieces, cudaStream_t st) {
  const size_t smem = static_cast<size_t>((p.R + 3) & ~3) * sizeof(float);
  const dim3 grid(p.H, pieces), block(256);
  if (p.D <= 32) return static_cast<int>(launch_kernel(delta_step_kernel<T, 4>, grid, block, smem, st, p));
  if (p.D <= 64) return static_cast<int>(launch_kernel(delta_step_kernel<T, 8>, grid, block, smem, st, p));
  return static_cast<int>(launch_kernel(delta_step_kernel<T, 16>, grid, block, smem, st, p));
}

template <int RPT>
static int launch_delta_scan(const DeltaParams& p, float* scratch, const int* slots, const int* cu, const int* reset,
                             int pieces, int row0, int N, cudaStream_t st) {
  constexpr int smem = 2 * kScanTok * (4 * 16 * RPT + kScanCta + 2) * 4;
  auto kern = delta_scan_kernel<RPT>;
  static bool configured[64] = {false};        // function attributes are per device
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) dev = 0;
  if (!configured[dev]) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    prefer_max_shared(kern);
    configured[dev] = true;
  }
  const int cbs = (p.D + kScanCta - 1) / kScanCta;
  return static_cast<int>(launch_kernel(kern, dim3(p.H * cbs, pieces), dim3(kScanCtaThreads), smem, st, p, scratch, slots, cu, reset, row0, N));
}

template <typename T>
static int delta_rule_typed(DeltaParams p, int pieces, int n_short, int rows, float* scratch, int mode, cudaStream_t st) {
  const bool small = p.D <= 128 && (p.R & ~3) < 2048;
  const bool vec = p.D % 4 == 0 && aligned_to(p.state, 16) && aligned_to(p.w2, 16);
  const bool w2_ok = p.R % 4 != 0 || aligned_to(p.w2, 16);
  if (mode == 1) return launch_delta_any<T>(p, pieces, st);
  if (n_short > 0) {
    const int rc = (small && vec) ? launch_delta_step<T>(p, n_short, st) : launch_delta_any<T>(p, n_short, st);
    if (rc) return rc;
  }
  const int np = pieces - n_short, N = rows - n_short;
  if (np <= 0 || N <= 0) return 0;
  DeltaParams q = p;
  q.slots += n_short, q.cu += n_short, q.reset += n_short;
  const size_t prep_smem = (static_cast<size_t>(kPrepTok) * ((p.R + 3) & ~3) + static_cast<size_t>(kPrepTok) * p.D) * sizeof(float);
  if (!small || !w2_ok || scratch == nullptr || prep_smem > 48 * 1024) return launch_delta_any<T>(q, np, st);
  const int tiles = (N + kPrepTok - 1) / kPrepTok;
  int rc = static_cast<int>(launch_kernel(delta_prep_kernel<T>, dim3(tiles, p.H), dim3(256), prep_smem, st, p, scratch, n_short, N));
  if (rc) return rc;
  if (p.D <= 32) rc = launch_delta_scan<2>(p, scratch, q.slots, q.cu, q.reset, np, n_short, N, st);
  else if (p.D <= 64) rc = launch_delta_scan<4>(p, scratch, q.slots, q.cu, q.reset, np, n_short, N, st);
  else rc = launch_delta_scan<8>(p, scratch, q.slots, q.cu, q.reset, np, n_short, N, st);
  if (rc) return rc;
  const long long warps = static_cast<long long>(N) * p.H;
  return static_cast<int>(launch_kernel(delta_post_kernel<T>, dim3(static_cast<unsigned>((warps + 7) / 8)), dim3(256), 0, st, p,
                                        static_cast<const float*>(scratch), n_short, N));
}

}  // namespace mx

using namespace mx;

extern "C" long long mx_delta_rule_scratch_floats(int tokens, int H, int D) {
  return static_cast<long long>(tokens) * H * (6ll * D + 2);
}

// A ragged batch of pieces (token rows cu[j] .. cu[j + 1] - 1 of proj and out, state slot slots[j], reset[j]
// starts from zero). The first n_short pieces hold exactly one token each; rows is the total number of
// token rows. offs: six element offsets of r, k, v, g, a, l in a row (host array). scratch:
// mx_delta_rule_scratch_floats(rows - n_short, H, D) floats, or NULL when every piece is short.
// mode 1 forces the kernel that covers any size.
extern "C" int mx_delta_rule(const void* proj, long long ld, const int* offs, const void* w2, const void* w0,
                             const void* a_bias, const void* norm_w, void* state, const void* slots, const void* cu,
                             const void* reset, void* out, void* scratch, int pieces, int n_short, int rows, int H, int D,
                             int R, float decay_scale, float unit_eps, float norm_eps, int fp32, int mode, void* stream) {
  if (pieces <= 0 || rows <= 0) return 0;
  if (offs == nullptr || H <= 0 || H > 65535 || D <= 0 || R <= 0 || pieces > 65535 || n_short < 0 || n_short > pieces) return -1;
  DeltaParams p{proj, ld, offs[0], offs[1], offs[2], offs[3], offs[4], offs[5], w2, static_cast<const float*>(w0),
                static_cast<const float*>(a_bias), static_cast<const float*>(norm_w), static_cast<float*>(state),
                static_cast<const int*>(slots), static_cast<const int*>(cu), static_cast<const int*>(reset), out, H, D, R,
                decay_scale, unit_eps, norm_eps};
  auto st = static_cast<cudaStream_t>(stream);
  auto* sc = static_cast<float*>(scratch);
  return fp32 ? delta_rule_typed<float>(p, pieces, n_short, rows, sc, mode, st)
              : delta_rule_typed<__nv_bfloat16>(p, pieces, n_short, rows, sc, mode, st);
}
