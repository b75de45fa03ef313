// Row kernels of layers that keep the residual stream in fp32 and normalise on both sides of a
// sub-layer, each for bf16 and fp32 activations:
//   embed_stream   h = scale * table[id], optionally normalised itself, plus a vector;  x = norm(h) or h as it is
//   stream_norm    h += norm(y) * layer scale, or y as it is;  h += a token's weighted experts, the embedding again, a
//                  vector;  x = norm(h) or h as it is                          (every part optional)
//   polynorm       a N(z) + b N(z^2) + c N(z^3) + e, N = division by the row's root mean square
//   glu_rows       gated activation of rows gate | up (SwiGLU, tanh-GeGLU, clipped SwiGLU)
//   softcap_rows   x <- cap tanh(x / cap) in fp32, in place
//   kv_append      k and v rows as projected into the paged pool
//   qk_norm_append per-head RMS norm of q and k, k and v rows into the paged pool (key and value heads
//                  may differ in width; no rotation)
// A norm weight w acts as (w_bias + w); all norm weights and layer scales are fp32 vectors, all
// arithmetic is fp32 and only the results are narrowed to the activation type.
#include "api.h"
#include "typed.cuh"

namespace mx {

// One CTA per row, V elements per access, up to VPT accesses per thread kept in registers: every
// input is read once and every output written once.
template <typename T, int V, int VPT, bool EX>
__device__ __forceinline__ void stream_step(const T* __restrict__ y, float* __restrict__ h, const int* __restrict__ rows,
                                            const float* __restrict__ post_w, const float* __restrict__ ls,
                                            const float* __restrict__ pre_w, T* __restrict__ x, int dim, float eps, float w_bias,
                                            const MxStreamExtras& ex) {
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.x;
  float* hr = h + static_cast<size_t>(rows != nullptr ? rows[row] : row) * dim;
  float hv[VPT][V];
  float s[1] = {0.f};
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < dim) load_v<V>(hr + c, hv[i]);
  }
  // hv += f * src[.] over this thread's columns
  const auto add = [&](const auto* src, float f) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * V;
      if (c < dim) {
        float a[V];
        load_v<V>(src + c, a);
#pragma unroll
        for (int e = 0; e < V; ++e) hv[i][e] = fmaf(f, a[e], hv[i][e]);
      }
    }
  };
  if (y != nullptr) {
    float yv[VPT][V];
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * V;
      if (c < dim) {
        load_v<V>(y + row * dim + c, yv[i]);
#pragma unroll
        for (int e = 0; e < V; ++e) s[0] += yv[i][e] * yv[i][e];
      }
    }
    float r = 1.f;
    if (post_w != nullptr) {
      block_sums<1>(s, red);
      r = 1.f / sqrtf(s[0] / dim + eps);
    }
    s[0] = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * V;
      if (c < dim) {
        float w[V], l[V];
        if (post_w != nullptr) load_v<V>(post_w + c, w);
        if (ls != nullptr) load_v<V>(ls + c, l);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const float b = post_w != nullptr ? yv[i][e] * r * (w_bias + w[e]) : yv[i][e];
          hv[i][e] += ls != nullptr ? b * l[e] : b;
        }
      }
    }
  }
  if (EX && ex.moe_ids != nullptr) {
#pragma unroll 4
    for (int k = 0; k < ex.moe_k; ++k) {
      const size_t pair = row * ex.moe_k + k;
      const T* src = ex.moe_ids[pair] >= ex.moe_experts ? static_cast<const T*>(ex.moe_x) + row * dim
                                                        : static_cast<const T*>(ex.moe_y) + static_cast<size_t>(ex.moe_inv[pair]) * dim;
      add(src, ex.moe_w[pair]);
    }
    if (ex.moe_shared != nullptr) add(static_cast<const T*>(ex.moe_shared) + row * dim, 1.f);
  }
  if (EX && ex.ids != nullptr) {
    const int id = ex.ids[row];
    if (id >= 0 && id < ex.vocab) add(static_cast<const T*>(ex.table) + static_cast<size_t>(id) * dim, ex.emb_scale);
  }
  if (EX && ex.vec != nullptr) add(ex.vec, 1.f);
  if (EX || y != nullptr) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * V;
      if (c < dim) store_v<V>(hr + c, hv[i]);
    }
  }
  if (x == nullptr) return;
  if (pre_w == nullptr) {                  // the sub-layer reads the stream itself
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * V;
      if (c < dim) store_v<V>(x + row * dim + c, hv[i]);
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < dim) {
#pragma unroll
      for (int e = 0; e < V; ++e) s[0] += hv[i][e] * hv[i][e];
    }
  }
  block_sums<1>(s, red);
  const float r = 1.f / sqrtf(s[0] / dim + eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < dim) {
      float w[V], o[V];
      load_v<V>(pre_w + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = hv[i][e] * r * (w_bias + w[e]);
      store_v<V>(x + row * dim + c, o);
    }
  }
}

template <typename T, int V, int VPT>
__global__ void __launch_bounds__(1024)
stream_norm_kernel(const T* __restrict__ y, float* __restrict__ h, const int* __restrict__ rows, const float* __restrict__ post_w,
                   const float* __restrict__ ls, const float* __restrict__ pre_w, T* __restrict__ x, int dim, float eps, float w_bias) {
  stream_step<T, V, VPT, false>(y, h, rows, post_w, ls, pre_w, x, dim, eps, w_bias, MxStreamExtras{});
}

template <typename T, int V, int VPT>
__global__ void __launch_bounds__(1024)
stream_sum_kernel(const T* __restrict__ y, float* __restrict__ h, const float* __restrict__ post_w, const float* __restrict__ ls,
                  const float* __restrict__ pre_w, T* __restrict__ x, int dim, float eps, float w_bias, const MxStreamExtras ex) {
  stream_step<T, V, VPT, true>(y, h, nullptr, post_w, ls, pre_w, x, dim, eps, w_bias, ex);
}

template <typename T, int V, int VPT>
__global__ void __launch_bounds__(1024)
embed_stream_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ h,
                    const float* __restrict__ own_w, const float* __restrict__ vec, const float* __restrict__ pre_w, T* __restrict__ x,
                    int dim, int vocab,
                    float scale, float eps, float w_bias) {
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.x;
  const int id = ids[row];
  const bool ok = id >= 0 && id < vocab;
  const T* tr = table + static_cast<size_t>(ok ? id : 0) * dim;
  float hv[VPT][V];
  float s[1] = {0.f};
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < dim) {
      load_v<V>(tr + c, hv[i]);
#pragma unroll
      for (int e = 0; e < V; ++e) hv[i][e] = ok ? hv[i][e] * scale : 0.f;
      if (own_w == nullptr && vec != nullptr) {
        float a[V];
        load_v<V>(vec + c, a);
#pragma unroll
        for (int e = 0; e < V; ++e) hv[i][e] += a[e];
      }
#pragma unroll
      for (int e = 0; e < V; ++e) s[0] += hv[i][e] * hv[i][e];
      if (own_w == nullptr) store_v<V>(h + row * dim + c, hv[i]);
    }
  }
  if (own_w != nullptr) {                  // the stream starts from the normalised embedding
    block_sums<1>(s, red);
    const float r = 1.f / sqrtf(s[0] / dim + eps);
    s[0] = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * V;
      if (c < dim) {
        float w[V], a[V];
        load_v<V>(own_w + c, w);
        if (vec != nullptr) load_v<V>(vec + c, a);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          hv[i][e] = hv[i][e] * r * (w_bias + w[e]) + (vec != nullptr ? a[e] : 0.f);
          s[0] += hv[i][e] * hv[i][e];
        }
        store_v<V>(h + row * dim + c, hv[i]);
      }
    }
  }
  if (x == nullptr) return;
  if (pre_w == nullptr) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * V;
      if (c < dim) store_v<V>(x + row * dim + c, hv[i]);
    }
    return;
  }
  block_sums<1>(s, red);
  const float r = 1.f / sqrtf(s[0] / dim + eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < dim) {
      float w[V], o[V];
      load_v<V>(pre_w + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = hv[i][e] * r * (w_bias + w[e]);
      store_v<V>(x + row * dim + c, o);
    }
  }
}

template <typename T, int V, int VPT>
__global__ void __launch_bounds__(1024)
polynorm_kernel(const T* __restrict__ z, const float* __restrict__ coef, T* __restrict__ out, int dim, float eps) {
  __shared__ float red[3 * 33];
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.x;
  float zv[VPT][V];
  float s[3] = {0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < dim) {
      load_v<V>(z + row * dim + c, zv[i]);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float q = zv[i][e] * zv[i][e];
        s[0] += q;
        s[1] += q * q;
        s[2] += q * q * q;
      }
    }
  }
  block_sums<3>(s, red);
  const float a = coef[0] / sqrtf(s[0] / dim + eps), b = coef[1] / sqrtf(s[1] / dim + eps),
              g = coef[2] / sqrtf(s[2] / dim + eps), e0 = coef[3];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < dim) {
      float o[V];
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = ((g * zv[i][e] + b) * zv[i][e] + a) * zv[i][e] + e0;
      store_v<V>(out + row * dim + c, o);
    }
  }
}

// Gated activation of rows gate [dim] | up [dim], `ld` elements apart; mode as MX_EPI_SWIGLU / GEGLU / CLIPPED_SWIGLU.
template <typename T, int V>
__global__ void __launch_bounds__(256)
glu_rows_kernel(const T* __restrict__ z, long long ld, T* __restrict__ out, int dim, int mode, float alpha, float limit) {
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.x;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= dim) return;
  float g[V], u[V];
  load_v<V>(z + row * ld + c, g);
  load_v<V>(z + row * ld + dim + c, u);
#pragma unroll
  for (int e = 0; e < V; ++e) {
    float a = g[e], b = u[e];
    if (mode == MX_EPI_GEGLU) {
      g[e] = 0.5f * a * (1.f + tanhf(0.7978845608028654f * (a + 0.044715f * a * a * a))) * b;
    } else {
      float k = 1.f;
      if (mode == MX_EPI_CLIPPED_SWIGLU) {
        a = fminf(a, limit);
        b = fminf(fmaxf(b, -limit), limit) + 1.f;
        k = alpha;
      }
      g[e] = a * sigmoid_f(k * a) * b;
    }
  }
  store_v<V>(out + row * dim + c, g);
}

template <int V>
__global__ void __launch_bounds__(256) softcap_rows_kernel(float* __restrict__ x, long long n, float cap) {
  pdl_trigger();
  pdl_wait();
  const float inv = 1.f / cap;
  for (long long i = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) * V; i < n; i += static_cast<long long>(gridDim.x) * blockDim.x * V) {
    float f[V];
    load_v<V>(x + i, f);
#pragma unroll
    for (int e = 0; e < V; ++e) f[e] = cap * tanhf(f[e] * inv);
    store_v<V>(x + i, f);
  }
}

// Rows of q | k | v (| more), `ld` elements apart. One CTA per token; a warp takes every eighth of the Hq
// query, Hkv key and Hkv value heads, kQkUnroll of them at a time so that their loads overlap: queries are
// normalised in place, keys normalised into the pool [blocks, Hkv, block_size, Dk], values copied into
// [blocks, Hkv, block_size, Dv]. Tokens with a negative slot append nothing. A lane keeps R groups of V
// elements in registers; wider heads read the rest twice.
constexpr int kQkUnroll = 3;

template <typename T, int V, int R>
__global__ void __launch_bounds__(256)
qk_norm_append_kernel(T* __restrict__ qkv, long long ld, const int* __restrict__ slots, T* __restrict__ k_pool,
                      T* __restrict__ v_pool, const float* __restrict__ qw, const float* __restrict__ kw, int Hq, int Hkv,
                      int Dk, int Dv, int block_size, float eps) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, per = Hq + 2 * Hkv, t = blockIdx.x;
  T* row = qkv + static_cast<size_t>(t) * ld;
  const int slot = slots[t];
  const int blk = slot >= 0 ? slot / block_size : 0, off = slot >= 0 ? slot - blk * block_size : 0;
  for (int h0 = warp; h0 < per; h0 += 8 * kQkUnroll) {
    T *src[kQkUnroll], *dst[kQkUnroll];
    const float* w[kQkUnroll];
    int D[kQkUnroll];                       // 0: nothing to do
    float f[kQkUnroll][R][V], s[kQkUnroll];
#pragma unroll
    for (int n = 0; n < kQkUnroll; ++n) {
      const int hd = h0 + 8 * n;
      src[n] = dst[n] = row, w[n] = nullptr, D[n] = 0, s[n] = 0.f;
      if (hd < Hq) {
        src[n] = dst[n] = row + static_cast<size_t>(hd) * Dk, w[n] = qw;
        D[n] = qw != nullptr ? Dk : 0;
      } else if (hd < per && slot >= 0) {
        const bool key = hd < Hq + Hkv;
        const int g = key ? hd - Hq : hd - Hq - Hkv;
        D[n] = key ? Dk : Dv;
        src[n] = row + static_cast<size_t>(Hq) * Dk + (key ? static_cast<size_t>(g) * Dk : static_cast<size_t>(Hkv) * Dk + static_cast<size_t>(g) * Dv);
        dst[n] = (key ? k_pool : v_pool) + ((static_cast<size_t>(blk) * Hkv + g) * block_size + off) * D[n];
        w[n] = key ? kw : nullptr;
      }
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int c = (lane + 32 * i) * V;
        if (c < D[n]) load_v<V>(src[n] + c, f[n][i]);
      }
    }
#pragma unroll
    for (int n = 0; n < kQkUnroll; ++n) {
      if (D[n] == 0) continue;              // (the same for the whole warp)
      float r = 1.f;
      if (w[n] != nullptr) {
#pragma unroll
        for (int i = 0; i < R; ++i) {
          const int c = (lane + 32 * i) * V;
          if (c < D[n]) {
#pragma unroll
            for (int e = 0; e < V; ++e) s[n] += f[n][i][e] * f[n][i][e];
          }
        }
        for (int c = (lane + 32 * R) * V; c < D[n]; c += 32 * V) {
          float g[V];
          load_v<V>(src[n] + c, g);
#pragma unroll
          for (int e = 0; e < V; ++e) s[n] += g[e] * g[e];
        }
        r = 1.f / sqrtf(warp_sum(s[n]) / D[n] + eps);
      }
      const auto emit = [&](int c, const float(&g)[V]) {
        float o[V], wv[V];
        if (w[n] != nullptr) load_v<V>(w[n] + c, wv);
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = w[n] != nullptr ? g[e] * r * wv[e] : g[e];
        store_v<V>(dst[n] + c, o);
      };
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int c = (lane + 32 * i) * V;
        if (c < D[n]) emit(c, f[n][i]);
      }
      for (int c = (lane + 32 * R) * V; c < D[n]; c += 32 * V) {
        float g[V];
        load_v<V>(src[n] + c, g);
        emit(c, g);
      }
    }
  }
}

// Keys and values as projected into the paged pool (no norm): one 16-byte group per thread over tokens and heads.
template <int BYTES>
__global__ void __launch_bounds__(256)
kv_append_kernel(const uint8_t* __restrict__ src, long long ld, const int* __restrict__ slots, uint8_t* __restrict__ k_pool,
                 uint8_t* __restrict__ v_pool, int n, int Hkv, int kb, int vb, int block_size) {      // ld, kb, vb: bytes
  pdl_trigger();
  pdl_wait();
  const int kg = Hkv * (kb / BYTES), per = kg + Hkv * (vb / BYTES);
  const unsigned i = blockIdx.x * 256u + threadIdx.x, t = i / per;
  if (t >= static_cast<unsigned>(n)) return;
  const int g = static_cast<int>(i - t * per), slot = slots[t];
  if (slot < 0) return;
  const bool key = g < kg;
  const int b = key ? kb : vb, j = key ? g : g - kg, head = j / (b / BYTES), at = (j - head * (b / BYTES)) * BYTES;
  const int blk = slot / block_size, off = slot - blk * block_size;
  const uint8_t* s = src + static_cast<size_t>(t) * ld + static_cast<size_t>(g) * BYTES;
  uint8_t* d = (key ? k_pool : v_pool) + ((static_cast<size_t>(blk) * Hkv + head) * block_size + off) * b + at;
  if constexpr (BYTES == 16) *reinterpret_cast<uint4*>(d) = *reinterpret_cast<const uint4*>(s);
  else *reinterpret_cast<uint16_t*>(d) = *reinterpret_cast<const uint16_t*>(s);
}

// Launch shape of a row kernel: groups of V elements per row -> threads and accesses per thread.
struct RowShape {
  int threads, vpt;
};
static RowShape row_shape(int dim, int v) {
  const int groups = (dim + v - 1) / v;
  int threads = (groups + 31) / 32 * 32;
  if (threads > 256) threads = groups > 8 * 256 ? 1024 : 256;
  if (threads < 64) threads = 64;
  const int need = (groups + threads - 1) / threads;
  return {threads, need <= 1 ? 1 : need <= 2 ? 2 : need <= 4 ? 4 : need <= 8 ? 8 : 0};
}

#define MX_ROW_DISPATCH(KERN, T, V, SHAPE, ROWS, STREAM, ...)                                                        \
  switch ((SHAPE).vpt) {                                                                                             \
    case 1: return static_cast<int>(launch_kernel(KERN<T, V, 1>, dim3(ROWS), dim3((SHAPE).threads), 0, STREAM, __VA_ARGS__)); \
    case 2: return static_cast<int>(launch_kernel(KERN<T, V, 2>, dim3(ROWS), dim3((SHAPE).threads), 0, STREAM, __VA_ARGS__)); \
    case 4: return static_cast<int>(launch_kernel(KERN<T, V, 4>, dim3(ROWS), dim3((SHAPE).threads), 0, STREAM, __VA_ARGS__)); \
    case 8: return static_cast<int>(launch_kernel(KERN<T, V, 8>, dim3(ROWS), dim3((SHAPE).threads), 0, STREAM, __VA_ARGS__)); \
    default: return -1;                                                                                              \
  }

template <typename T>
static int stream_norm_typed(const void* y, void* h, const void* rows, const float* post_w, const float* ls, const float* pre_w,
                             void* x, int n, int dim, float eps, float w_bias, const MxStreamExtras* ex, bool vec, cudaStream_t st) {
  const T* yp = static_cast<const T*>(y);
  const int* rp = static_cast<const int*>(rows);
  const RowShape sh = row_shape(dim, vec ? 4 : 1);
  auto *hp = static_cast<float*>(h);
  auto *xp = static_cast<T*>(x);
  if (ex != nullptr) {
    if (vec) MX_ROW_DISPATCH(stream_sum_kernel, T, 4, sh, n, st, yp, hp, post_w, ls, pre_w, xp, dim, eps, w_bias, *ex)
    MX_ROW_DISPATCH(stream_sum_kernel, T, 1, sh, n, st, yp, hp, post_w, ls, pre_w, xp, dim, eps, w_bias, *ex)
  }
  if (vec) MX_ROW_DISPATCH(stream_norm_kernel, T, 4, sh, n, st, yp, hp, rp, post_w, ls, pre_w, xp, dim, eps, w_bias)
  MX_ROW_DISPATCH(stream_norm_kernel, T, 1, sh, n, st, yp, hp, rp, post_w, ls, pre_w, xp, dim, eps, w_bias)
}

template <typename T>
static int embed_stream_typed(const int* ids, const void* table, void* h, const float* own_w, const float* add, const float* pre_w, void* x, int n, int dim, int vocab,
                              float scale, float eps, float w_bias, bool vec, cudaStream_t st) {
  const T* tp = static_cast<const T*>(table);
  if (vec) {
    const RowShape sh = row_shape(dim, 4);
    MX_ROW_DISPATCH(embed_stream_kernel, T, 4, sh, n, st, ids, tp, static_cast<float*>(h), own_w, add, pre_w, static_cast<T*>(x), dim, vocab, scale, eps, w_bias)
  }
  const RowShape sh = row_shape(dim, 1);
  MX_ROW_DISPATCH(embed_stream_kernel, T, 1, sh, n, st, ids, tp, static_cast<float*>(h), own_w, add, pre_w, static_cast<T*>(x), dim, vocab, scale, eps, w_bias)
}

template <typename T>
static int polynorm_typed(const void* z, const float* coef, void* out, int n, int dim, float eps, bool vec, cudaStream_t st) {
  const T* zp = static_cast<const T*>(z);
  if (vec) {
    const RowShape sh = row_shape(dim, 4);
    MX_ROW_DISPATCH(polynorm_kernel, T, 4, sh, n, st, zp, coef, static_cast<T*>(out), dim, eps)
  }
  const RowShape sh = row_shape(dim, 1);
  MX_ROW_DISPATCH(polynorm_kernel, T, 1, sh, n, st, zp, coef, static_cast<T*>(out), dim, eps)
}

template <typename T>
static int qk_norm_append_typed(void* qkv, long long ld, const int* slots, void* k_pool, void* v_pool, const float* qw,
                                const float* kw, int n, int Hq, int Hkv, int Dk, int Dv, int bs, float eps, bool vec,
                                cudaStream_t st) {
  const dim3 grid(n), block(256);
  T *qp = static_cast<T*>(qkv), *kp = static_cast<T*>(k_pool), *vp = static_cast<T*>(v_pool);
  auto kern = !vec ? qk_norm_append_kernel<T, 1, 4> : (Dk <= 128 && Dv <= 128) ? qk_norm_append_kernel<T, 4, 1> : qk_norm_append_kernel<T, 4, 2>;
  return static_cast<int>(launch_kernel(kern, grid, block, 0, st, qp, ld, slots, kp, vp, qw, kw, Hq, Hkv, Dk, Dv, bs, eps));
}

}  // namespace mx

using namespace mx;

// fp32: 1 = fp32 activations, 0 = bf16. y / rows / post_w / ls / extras / x may be NULL (no branch to add, identity row
// map, the branch is not normalised, no layer scale, nothing else to add, no output); x with pre_w == NULL receives the stream itself.
extern "C" int mx_stream_norm(const void* y, void* h, const void* rows, const void* post_w, const void* ls,
                              const void* pre_w, void* x, int n, int dim, float eps, float w_bias, int fp32,
                              const MxStreamExtras* extras, void* stream) {
  if (n <= 0 || dim <= 0) return 0;
  const MxStreamExtras ex = extras != nullptr ? *extras : MxStreamExtras{};
  if (h == nullptr || (rows != nullptr && (y != nullptr || extras != nullptr))) return -1;
  if (ex.moe_ids != nullptr && (ex.moe_x == nullptr || ex.moe_y == nullptr || ex.moe_inv == nullptr || ex.moe_w == nullptr)) return -1;
  if (ex.ids != nullptr && (ex.table == nullptr || ex.vec == nullptr)) return -1;
  const size_t ab = fp32 ? 16 : 8;
  const bool vec = dim % 4 == 0 && aligned_to(y, ab) && aligned_to(x, ab) && aligned_to(h, 16) && aligned_to(post_w, 16) &&
                   aligned_to(ls, 16) && aligned_to(pre_w, 16) && aligned_to(ex.moe_y, ab) && aligned_to(ex.moe_x, ab) &&
                   aligned_to(ex.moe_shared, ab) && aligned_to(ex.table, ab) && aligned_to(ex.vec, 16);
  auto st = static_cast<cudaStream_t>(stream);
  const float *pw = static_cast<const float*>(post_w), *lp = static_cast<const float*>(ls), *nw = static_cast<const float*>(pre_w);
  return fp32 ? stream_norm_typed<float>(y, h, rows, pw, lp, nw, x, n, dim, eps, w_bias, extras, vec, st)
              : stream_norm_typed<__nv_bfloat16>(y, h, rows, pw, lp, nw, x, n, dim, eps, w_bias, extras, vec, st);
}

extern "C" int mx_embed_stream(const void* ids, const void* table, void* h, const void* own_w, const void* add, const void* pre_w,
                               void* x, int n, int dim, int vocab, float scale, float eps, float w_bias, int fp32, void* stream) {
  if (n <= 0 || dim <= 0) return 0;
  const size_t ab = fp32 ? 16 : 8;
  const bool vec = dim % 4 == 0 && aligned_to(table, ab) && aligned_to(x, ab) && aligned_to(h, 16) && aligned_to(own_w, 16) &&
                   aligned_to(pre_w, 16) && aligned_to(add, 16);
  auto st = static_cast<cudaStream_t>(stream);
  const float *ow = static_cast<const float*>(own_w), *av = static_cast<const float*>(add), *nw = static_cast<const float*>(pre_w);
  const int* ip = static_cast<const int*>(ids);
  return fp32 ? embed_stream_typed<float>(ip, table, h, ow, av, nw, x, n, dim, vocab, scale, eps, w_bias, vec, st)
              : embed_stream_typed<__nv_bfloat16>(ip, table, h, ow, av, nw, x, n, dim, vocab, scale, eps, w_bias, vec, st);
}

extern "C" int mx_polynorm(const void* z, const void* coef, void* out, int n, int dim, float eps, int fp32, void* stream) {
  if (n <= 0 || dim <= 0) return 0;
  const size_t ab = fp32 ? 16 : 8;
  const bool vec = dim % 4 == 0 && aligned_to(z, ab) && aligned_to(out, ab);
  auto st = static_cast<cudaStream_t>(stream);
  const float* cp = static_cast<const float*>(coef);
  return fp32 ? polynorm_typed<float>(z, cp, out, n, dim, eps, vec, st)
              : polynorm_typed<__nv_bfloat16>(z, cp, out, n, dim, eps, vec, st);
}

extern "C" int mx_qk_norm_append(void* qkv, long long ld, const void* slots, void* k_pool, void* v_pool, const void* qw,
                                 const void* kw, int n, int Hq, int Hkv, int Dk, int Dv, int block_size, float eps,
                                 int fp32, void* stream) {
  if (n <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || Dk <= 0 || Dv <= 0 || block_size <= 0) return -1;
  if (qw == nullptr && kw == nullptr) {
    const int es = fp32 ? 4 : 2, kb = Dk * es, vb = Dv * es;
    const auto* src = static_cast<const uint8_t*>(qkv) + static_cast<size_t>(Hq) * Dk * es;
    const bool wide = kb % 16 == 0 && vb % 16 == 0 && ld * es % 16 == 0 && aligned_to(src, 16) && aligned_to(k_pool, 16) && aligned_to(v_pool, 16);
    const long long groups = static_cast<long long>(n) * Hkv * (kb + vb) / (wide ? 16 : 2);
    if (groups > 0x7fffffffll) return -1;
    return static_cast<int>(launch_kernel(wide ? kv_append_kernel<16> : kv_append_kernel<2>, dim3(static_cast<unsigned>((groups + 255) / 256)),
                                          dim3(256), 0, static_cast<cudaStream_t>(stream), src, ld * es, static_cast<const int*>(slots),
                                          static_cast<uint8_t*>(k_pool), static_cast<uint8_t*>(v_pool), n, Hkv, kb, vb, block_size));
  }
  const size_t ab = fp32 ? 16 : 8;
  const bool vec = Dk % 4 == 0 && Dv % 4 == 0 && ld % 4 == 0 && aligned_to(qkv, ab) && aligned_to(k_pool, ab) &&
                   aligned_to(v_pool, ab) && aligned_to(qw, 16) && aligned_to(kw, 16);
  auto st = static_cast<cudaStream_t>(stream);
  const int* sp = static_cast<const int*>(slots);
  const float *q = static_cast<const float*>(qw), *k = static_cast<const float*>(kw);
  return fp32 ? qk_norm_append_typed<float>(qkv, ld, sp, k_pool, v_pool, q, k, n, Hq, Hkv, Dk, Dv, block_size, eps, vec, st)
              : qk_norm_append_typed<__nv_bfloat16>(qkv, ld, sp, k_pool, v_pool, q, k, n, Hq, Hkv, Dk, Dv, block_size, eps, vec, st);
}

// z rows gate | up (2 dim elements, ld apart) -> out rows of dim.
extern "C" int mx_glu_rows(const void* z, long long ld, void* out, int n, int dim, int mode, float alpha, float limit, int fp32,
                           void* stream) {
  if (n <= 0 || dim <= 0) return 0;
  if (mode < MX_EPI_SWIGLU || mode > MX_EPI_CLIPPED_SWIGLU || dim > 65535 * 256) return -1;
  const size_t ab = fp32 ? 16 : 8;
  const bool vec = dim % 4 == 0 && ld % 4 == 0 && aligned_to(z, ab) && aligned_to(out, ab);
  auto st = static_cast<cudaStream_t>(stream);
  const dim3 grid(n, (dim + (vec ? 1023 : 255)) / (vec ? 1024 : 256)), block(256);
#define MX_GLU(T, V)                                                                                                    \
  return static_cast<int>(launch_kernel(glu_rows_kernel<T, V>, grid, block, 0, st, static_cast<const T*>(z), ld,        \
                                        static_cast<T*>(out), dim, mode, alpha, limit))
  if (fp32) {
    if (vec) MX_GLU(float, 4);
    MX_GLU(float, 1);
  }
  if (vec) MX_GLU(__nv_bfloat16, 4);
  MX_GLU(__nv_bfloat16, 1);
#undef MX_GLU
}

// x (fp32, n contiguous values) <- cap tanh(x / cap).
extern "C" int mx_softcap_rows(void* x, long long n, float cap, void* stream) {
  if (n <= 0) return 0;
  if (!(cap > 0.f)) return -1;
  const bool vec = n % 4 == 0 && aligned_to(x, 16);
  const long long blocks = (n + (vec ? 1023 : 255)) / (vec ? 1024 : 256);
  return static_cast<int>(launch_kernel(vec ? softcap_rows_kernel<4> : softcap_rows_kernel<1>, dim3(static_cast<unsigned>(blocks < 4096 ? blocks : 4096)), dim3(256), 0,
                                        static_cast<cudaStream_t>(stream), static_cast<float*>(x), n, cap));
}
