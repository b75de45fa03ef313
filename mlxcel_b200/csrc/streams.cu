// Row kernels of layers with several residual streams, for bf16 and fp32 activations; all arithmetic is fp32:
//   streams_step     one step between two sub-layers (see MxStreamsStep): the streams take up what the last sub-layer returned and
//                    are mixed, the next one's input is gathered and layer-normalised; for rows that are pieces of one token
//                    (decode) also convolved over time. Every stream is read and written once
//   streams_conv     x = n + causal convolution of n per channel, over prompt portions
//   layer_norm_rows  layer norm with weight and bias
#include "api.h"
#include "typed.cuh"

namespace mx {

constexpr int kMaxStreams = 16;

// One CTA per row; a thread takes VPT groups of V columns and keeps the sub-layer's input in registers. S_ streams, or up to
// kMaxStreams of them (S_ == 0).
template <typename T, int V, int VPT, int S_>
__global__ void __launch_bounds__(512) streams_step_kernel(const MxStreamsStep p) {
  constexpr int SM = S_ > 0 ? S_ : kMaxStreams;
  const int S = S_ > 0 ? S_ : p.streams;
  __shared__ float red[33], mix_s[SM * SM], out_s[SM], in_s[SM];
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) mix_s[i] = p.mix != nullptr ? p.mix[i] : 0.f;
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    out_s[i] = p.w_out != nullptr ? p.w_out[i] : 0.f;
    in_s[i] = p.w_in != nullptr ? p.w_in[i] : 1.f;
  }
  pdl_trigger();
  pdl_wait();
  __syncthreads();
  const int row = blockIdx.x, dim = p.dim;
  float* xr = p.xs + static_cast<size_t>(row) * S * dim;
  const T* er = nullptr;                                   // the token's embedding
  bool known = false;
  if (p.ids != nullptr) {
    const int id = p.ids[row];
    known = id >= 0 && id < p.vocab;
    er = static_cast<const T*>(p.table) + static_cast<size_t>(known ? id : 0) * dim;
  }
  const int K = p.taps;
  const bool single = row < p.n_short;                     // a piece of one token
  const int slot = single ? p.slots[row] : 0;
  float* tail = single && slot >= 0 ? p.tail + static_cast<size_t>(slot) * (K - 1) * dim : nullptr;
  if (tail != nullptr)                                     // (its state is needed behind the norm)
    for (int c = threadIdx.x * 32; c < (K - 1) * dim; c += blockDim.x * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(tail + c));
  float u[VPT][V], s[1] = {0.f};
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) u[i][e] = 0.f;
    if (c >= dim) continue;
    float x[SM][V], y[V];
    if (p.ids != nullptr) {
      load_v<V>(er + c, y);
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = known ? y[e] * p.emb_scale : 0.f;
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= S) break;
        store_v<V>(xr + static_cast<size_t>(t) * dim + c, y);
#pragma unroll
        for (int e = 0; e < V; ++e) u[i][e] = fmaf(in_s[t], y[e], u[i][e]);
      }
    } else {
#pragma unroll
      for (int t = 0; t < SM; ++t)
        if (t < S) load_v<V>(xr + static_cast<size_t>(t) * dim + c, x[t]);
      if (p.moe_y != nullptr) {
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = 0.f;
#pragma unroll 4
        for (int k = 0; k < p.moe_k; ++k) {
          const size_t pair = static_cast<size_t>(row) * p.moe_k + k;
          const float w = p.moe_w[pair];
          float a[V];
          load_v<V>(static_cast<const T*>(p.moe_y) + static_cast<size_t>(p.moe_inv[pair]) * dim + c, a);
#pragma unroll
          for (int e = 0; e < V; ++e) y[e] = fmaf(w, a[e], y[e]);
        }
      } else {
        load_v<V>(static_cast<const T*>(p.y) + static_cast<size_t>(row) * dim + c, y);
      }
      if (p.bias != nullptr) {
        float a[V];
        load_v<V>(p.bias + c, a);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] += a[e];
      }
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= S) break;
        float n[V];
#pragma unroll
        for (int e = 0; e < V; ++e) n[e] = out_s[t] * y[e];
#pragma unroll
        for (int f = 0; f < SM; ++f) {
          if (f >= S) break;
          const float m = mix_s[f * S + t];
#pragma unroll
          for (int e = 0; e < V; ++e) n[e] = fmaf(m, x[f][e], n[e]);
        }
        if (p.sum == nullptr) store_v<V>(xr + static_cast<size_t>(t) * dim + c, n);
#pragma unroll
        for (int e = 0; e < V; ++e) u[i][e] = fmaf(in_s[t], n[e], u[i][e]);
      }
      if (p.sum != nullptr) store_v<V>(p.sum + static_cast<size_t>(row) * dim + c, u[i]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) s[0] += u[i][e];
  }
  if (p.x == nullptr) return;
  block_sums<1>(s, red);
  const float mean = s[0] / dim;
  s[0] = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    if ((threadIdx.x + i * blockDim.x) * V >= dim) continue;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      u[i][e] -= mean;
      s[0] = fmaf(u[i][e], u[i][e], s[0]);
    }
  }
  block_sums<1>(s, red);
  const float r = 1.f / sqrtf(s[0] / dim + p.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c >= dim) continue;
    float w[V], b[V], n[V];
    load_v<V>(p.norm_w + c, w);
    load_v<V>(p.norm_b + c, b);
#pragma unroll
    for (int e = 0; e < V; ++e) n[e] = fmaf(u[i][e] * r, w[e], b[e]);
    if (!single && K > 1) {
      store_v<V>(p.normed + static_cast<size_t>(row - p.n_short) * dim + c, n);
      continue;
    }
    float o[V];
    load_v<V>(p.taps_w + static_cast<size_t>(K - 1) * dim + c, w);
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = fmaf(w[e], n[e], n[e]);
    if (tail != nullptr) {
      for (int k = 0; k < K - 1; ++k) {                    // the state moves up by one
        float a[V];
        load_v<V>(tail + static_cast<size_t>(k) * dim + c, a);
        load_v<V>(p.taps_w + static_cast<size_t>(k) * dim + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = fmaf(w[e], a[e], o[e]);
        if (k > 0) store_v<V>(tail + static_cast<size_t>(k - 1) * dim + c, a);
      }
      if (K > 1) store_v<V>(tail + static_cast<size_t>(K - 2) * dim + c, n);
    }
    store_v<V>(static_cast<T*>(p.x) + static_cast<size_t>(row) * dim + c, o);
  }
}

struct ConvParams {
  const float* n;            // rows of this call, row0 taken off
  const float* w;            // [taps, dim]
  float* tail;               // [slots, taps - 1, dim]
  const int* slots;
  const int* cu;             // rows of the whole batch
  const int* reset;
  void* x;
  int row0, dim, taps, run;
};

// A thread takes V channels of `run` tokens of one piece (run >= taps - 1, so that only a piece's first run looks back into
// the state). That run's threads also leave the new state: the piece's last taps - 1 inputs.
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(128) streams_conv_kernel(const ConvParams p) {
  pdl_trigger();
  pdl_wait();
  const int K = TAPS > 0 ? TAPS : p.taps, dim = p.dim, c = (blockIdx.y * blockDim.x + threadIdx.x) * V, j = blockIdx.z;
  const int t0 = p.cu[j] - p.row0, t1 = p.cu[j + 1] - p.row0, r0 = t0 + blockIdx.x * p.run, r1 = min(t1, r0 + p.run);
  if (c >= dim || r0 >= t1) return;
  const int slot = p.slots[j];
  const bool fresh = slot < 0 || p.reset[j] != 0;
  float* tail = p.tail + static_cast<size_t>(max(slot, 0)) * (K - 1) * dim + c;
  const float* n = p.n + c;
  T* x = static_cast<T*>(p.x) + static_cast<size_t>(p.row0) * dim + c;
  const auto input = [&](int t, float (&a)[V]) {           // of token t, also before the piece
    if (t >= t0) load_v<V>(n + static_cast<size_t>(t) * dim, a);
    else if (!fresh) load_v<V>(tail + static_cast<size_t>(K - 1 + t - t0) * dim, a);
    else {
#pragma unroll
      for (int e = 0; e < V; ++e) a[e] = 0.f;
    }
  };
  if constexpr (TAPS > 0) {
    constexpr int B = 4;                                   // rows requested at a time
    float w[TAPS][V], h[TAPS][V];
#pragma unroll
    for (int k = 0; k < TAPS; ++k) load_v<V>(p.w + static_cast<size_t>(k) * dim + c, w[k]);
#pragma unroll
    for (int k = 1; k < TAPS; ++k) input(r0 - TAPS + k, h[k]);
    for (int b0 = r0; b0 < r1; b0 += B) {
      float in[B][V];
#pragma unroll
      for (int b = 0; b < B; ++b) load_v<V>(n + static_cast<size_t>(min(b0 + b, r1 - 1)) * dim, in[b]);
#pragma unroll
      for (int b = 0; b < B; ++b) {
        if (b0 + b >= r1) break;
        float o[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
          o[e] = in[b][e];
#pragma unroll
          for (int k = 0; k < TAPS; ++k) {
            h[k][e] = k + 1 < TAPS ? h[k + 1 < TAPS ? k + 1 : k][e] : in[b][e];
            o[e] = fmaf(w[k][e], h[k][e], o[e]);
          }
        }
        store_v<V>(x + static_cast<size_t>(b0 + b) * dim, o);
      }
    }
  } else {
    for (int t = r0; t < r1; ++t) {
      float o[V];
      load_v<V>(n + static_cast<size_t>(t) * dim, o);
      for (int k = 0; k < K; ++k) {
        float a[V], w[V];
        input(t - K + 1 + k, a);
        load_v<V>(p.w + static_cast<size_t>(k) * dim + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = fmaf(w[e], a[e], o[e]);
      }
      store_v<V>(x + static_cast<size_t>(t) * dim, o);
    }
  }
  if (blockIdx.x == 0 && slot >= 0)
    for (int k = 0; k < K - 1; ++k) {                      // (entry k comes from a later one, or from the piece)
      float a[V];
      input(t1 - (K - 1) + k, a);
      store_v<V>(tail + static_cast<size_t>(k) * dim, a);
    }
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
layer_norm_rows_kernel(const float* __restrict__ h, const int* __restrict__ rows, const float* __restrict__ w, const float* __restrict__ b,
                       T* __restrict__ out, int dim, float eps) {
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.x;
  const float* hr = h + static_cast<size_t>(rows != nullptr ? rows[row] : row) * dim;
  float s[1] = {0.f}, a[V], g[V], z[V];
  for (int c = threadIdx.x * V; c < dim; c += blockDim.x * V) {
    load_v<V>(hr + c, a);
#pragma unroll
    for (int e = 0; e < V; ++e) s[0] += a[e];
  }
  block_sums<1>(s, red);
  const float mean = s[0] / dim;
  s[0] = 0.f;
  for (int c = threadIdx.x * V; c < dim; c += blockDim.x * V) {
    load_v<V>(hr + c, a);
#pragma unroll
    for (int e = 0; e < V; ++e) s[0] = fmaf(a[e] - mean, a[e] - mean, s[0]);
  }
  block_sums<1>(s, red);
  const float r = 1.f / sqrtf(s[0] / dim + eps);
  for (int c = threadIdx.x * V; c < dim; c += blockDim.x * V) {
    load_v<V>(hr + c, a);
    load_v<V>(w + c, g);
    load_v<V>(b + c, z);
#pragma unroll
    for (int e = 0; e < V; ++e) a[e] = fmaf((a[e] - mean) * r, g[e], z[e]);
    store_v<V>(out + row * dim + c, a);
  }
}

template <typename T, int V, int S>
static int launch_step(const MxStreamsStep& p, cudaStream_t st) {
  const int groups = (p.dim + V - 1) / V;
  int threads = (groups + 31) / 32 * 32;
  // (few rows: all of a row's accesses at once; many: more rows per SM)
  const int most = p.rows <= 296 || groups > 256 * 8 ? 512 : 256;
  threads = threads < 64 ? 64 : threads <= most ? threads : most;
  const int need = (groups + threads - 1) / threads;
  const dim3 grid(p.rows), block(threads);
  if (need <= 1) return static_cast<int>(launch_kernel(streams_step_kernel<T, V, 1, S>, grid, block, 0, st, p));
  if (need <= 2) return static_cast<int>(launch_kernel(streams_step_kernel<T, V, 2, S>, grid, block, 0, st, p));
  if (need <= 4) return static_cast<int>(launch_kernel(streams_step_kernel<T, V, 4, S>, grid, block, 0, st, p));
  if (need <= 16) return static_cast<int>(launch_kernel(streams_step_kernel<T, V, 16, S>, grid, block, 0, st, p));
  return -1;
}

template <typename T>
static int streams_step_typed(const MxStreamsStep& p, bool vec, cudaStream_t st) {
  if (!vec) return launch_step<T, 1, 0>(p, st);
  switch (p.streams) {
    case 2: return launch_step<T, 4, 2>(p, st);
    case 4: return launch_step<T, 4, 4>(p, st);
    default: return launch_step<T, 4, 0>(p, st);
  }
}

template <typename T, int V>
static int launch_conv(const ConvParams& p, dim3 grid, cudaStream_t st) {
  const dim3 block(128);
  switch (p.taps) {
    case 2: return static_cast<int>(launch_kernel(streams_conv_kernel<T, V, 2>, grid, block, 0, st, p));
    case 3: return static_cast<int>(launch_kernel(streams_conv_kernel<T, V, 3>, grid, block, 0, st, p));
    case 4: return static_cast<int>(launch_kernel(streams_conv_kernel<T, V, 4>, grid, block, 0, st, p));
    default: return static_cast<int>(launch_kernel(streams_conv_kernel<T, V, 0>, grid, block, 0, st, p));
  }
}

}  // namespace mx

using namespace mx;

extern "C" int mx_streams_step(const MxStreamsStep* step, int fp32, void* stream) {
  const MxStreamsStep& p = *step;
  if (p.rows <= 0 || p.dim <= 0) return 0;
  if (p.xs == nullptr || p.streams < 1 || p.streams > kMaxStreams) return -1;
  if (p.ids != nullptr ? p.table == nullptr : (p.mix == nullptr || p.w_out == nullptr || (p.y == nullptr) == (p.moe_y == nullptr))) return -1;
  if (p.moe_y != nullptr && (p.moe_inv == nullptr || p.moe_w == nullptr || p.moe_k < 1)) return -1;
  if ((p.x == nullptr) == (p.sum == nullptr) || (p.sum != nullptr && (p.ids != nullptr || p.w_in != nullptr))) return -1;
  if (p.x != nullptr && (p.w_in == nullptr || p.norm_w == nullptr || p.norm_b == nullptr || p.taps_w == nullptr || p.taps < 1)) return -1;
  if (p.x != nullptr && p.n_short > 0 && (p.slots == nullptr || (p.taps > 1 && p.tail == nullptr))) return -1;
  if (p.x != nullptr && p.n_short < p.rows && p.taps > 1 && p.normed == nullptr) return -1;
  const size_t ab = fp32 ? 16 : 8;
  const bool vec = p.dim % 4 == 0 && aligned_to(p.xs, 16) && aligned_to(p.table, ab) && aligned_to(p.y, ab) && aligned_to(p.moe_y, ab) &&
                   aligned_to(p.bias, 16) && aligned_to(p.norm_w, 16) && aligned_to(p.norm_b, 16) && aligned_to(p.taps_w, 16) &&
                   aligned_to(p.tail, 16) && aligned_to(p.x, ab) && aligned_to(p.normed, 16) && aligned_to(p.sum, 16);
  auto st = static_cast<cudaStream_t>(stream);
  return fp32 ? streams_step_typed<float>(p, vec, st) : streams_step_typed<__nv_bfloat16>(p, vec, st);
}

// Pieces cu[j] .. cu[j + 1] - 1 (rows of the whole batch, of which n holds those from row0 on), state slot slots[j], reset[j] starts from
// zero; `longest` bounds their length. x [rows, dim].
extern "C" int mx_streams_conv(const void* n, const void* w, void* tail, const void* slots, const void* cu, const void* reset, void* x,
                               int pieces, int row0, int rows, int dim, int taps, int longest, int fp32, void* stream) {
  if (pieces <= 0 || rows <= row0 || dim <= 0) return 0;
  if (taps < 2 || longest < 1 || pieces > 65535) return -1;
  const size_t ab = fp32 ? 16 : 8;
  const bool vec = dim % 4 == 0 && aligned_to(n, 16) && aligned_to(w, 16) && aligned_to(tail, 16) && aligned_to(x, ab);
  const ConvParams p{static_cast<const float*>(n), static_cast<const float*>(w), static_cast<float*>(tail), static_cast<const int*>(slots),
                     static_cast<const int*>(cu), static_cast<const int*>(reset), x, row0, dim, taps, taps - 1 > 16 ? taps - 1 : 16};
  const int per = 128 * (vec ? 4 : 1);
  const dim3 grid((longest + p.run - 1) / p.run, (dim + per - 1) / per, pieces);
  auto st = static_cast<cudaStream_t>(stream);
  if (fp32) return vec ? launch_conv<float, 4>(p, grid, st) : launch_conv<float, 1>(p, grid, st);
  return vec ? launch_conv<__nv_bfloat16, 4>(p, grid, st) : launch_conv<__nv_bfloat16, 1>(p, grid, st);
}

// Row r of out is the norm of row rows[r] of h (or r). w and b fp32.
extern "C" int mx_layer_norm_rows(const void* h, const void* rows, const void* w, const void* b, void* out, int n, int dim, float eps, int fp32,
                                  void* stream) {
  if (n <= 0 || dim <= 0) return 0;
  const bool vec = dim % 4 == 0 && aligned_to(h, 16) && aligned_to(w, 16) && aligned_to(b, 16) && aligned_to(out, fp32 ? 16 : 8);
  const auto *hp = static_cast<const float*>(h), *wp = static_cast<const float*>(w), *bp = static_cast<const float*>(b);
  const int* rp = static_cast<const int*>(rows);
  auto st = static_cast<cudaStream_t>(stream);
  if (fp32)
    return static_cast<int>(launch_kernel(vec ? layer_norm_rows_kernel<float, 4> : layer_norm_rows_kernel<float, 1>, dim3(n), dim3(256), 0, st, hp,
                                          rp, wp, bp, static_cast<float*>(out), dim, eps));
  return static_cast<int>(launch_kernel(vec ? layer_norm_rows_kernel<__nv_bfloat16, 4> : layer_norm_rows_kernel<__nv_bfloat16, 1>, dim3(n), dim3(256),
                                        0, st, hp, rp, wp, bp, static_cast<__nv_bfloat16*>(out), dim, eps));
}
