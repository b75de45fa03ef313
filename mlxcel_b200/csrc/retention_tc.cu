// Retention of prompt portions in chunks on the 5th-generation tensor cores (tcgen05 + TMEM), bf16 rows.
//
// With decay g and the state S_0 before a chunk of n tokens (numbered from 0):
//   o_i = g^(i + 1) S_0^T q_i + sum_{j <= i} g^(i - j) (q_i . k_j) v_j          S_n = g^n S_0 + sum_j g^(n - 1 - j) k_j v_j^T
// A CTA owns one head (and 128 of its value columns) of one piece and walks its chunks of 128 tokens; per chunk four products:
//   scores   A = q k^T          read-out  Q = q S_0          values  O = (A masked by the decays) v          state  dS^T = v^T (decayed k)
// Everything that enters them is fp32 (rotated queries and keys, the state, decayed scores and keys) and is fed to the tensor
// cores as the sum of two bf16 terms (rounded value and remainder), the product of the two remainders left out: 16 bits of each
// operand, accumulated in fp32. The state itself stays in fp32 registers (thread: one value column, half of the key channels) and is
// written to shared memory as the next chunk's operand.
//
// The eight warps work in step: rotate and stage the chunk's rows, wait for scores and read-out, mask the scores (into the
// queries' place) and decay the keys (in place), wait for the values and finish the rows (norm, gate), wait for the state. Every
// wait is bounded and reports through the status word.
#include "api.h"
#include "retention.cuh"

namespace mx {

constexpr int kRtThreads = 256;
constexpr int kRtSub = 128 * 128;                          // bytes of a [128 rows][64 columns] sub-tile
constexpr int kRtTerm = 2 * kRtSub;                        // bytes of a [128][128] bf16 tile
constexpr int kRtSmem = 1024 + 7 * kRtTerm + 2048;         // q, k, state as two terms each, v; decays, sums, barriers
constexpr int kErrRetention = 501;
static_assert(kRtSmem <= 227 * 1024, "shared memory");

// Cosine and sine of every token's angles.
__global__ void __launch_bounds__(256)
retention_angles_kernel(const int* __restrict__ positions, const float* __restrict__ inv_freq, float2* __restrict__ cs, int half, int N) {
  pdl_trigger();
  pdl_wait();
  const unsigned i = blockIdx.x * 256u + threadIdx.x, n = i / half;
  if (n >= static_cast<unsigned>(N)) return;
  float s, c;
  sincosf(static_cast<float>(positions[n]) * inv_freq[i - n * half], &s, &c);
  cs[i] = make_float2(c, s);
}

__device__ __forceinline__ void unpack8(const uint4& a, float (&f)[8]) {
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) f[2 * i] = bf16_lo(w[i]), f[2 * i + 1] = bf16_hi(w[i]);
}
// Eight values as two bf16 terms at the same place of two tiles.
__device__ __forceinline__ void store_terms(uint8_t* hi, const float (&f)[8]) {
  uint32_t a[4], b[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    a[i] = pack_bf16(f[2 * i], f[2 * i + 1]);
    b[i] = pack_bf16(f[2 * i] - bf16_lo(a[i]), f[2 * i + 1] - bf16_hi(a[i]));
  }
  *reinterpret_cast<uint4*>(hi) = make_uint4(a[0], a[1], a[2], a[3]);
  *reinterpret_cast<uint4*>(hi + kRtTerm) = make_uint4(b[0], b[1], b[2], b[3]);
}
// Byte of 16-byte group ch (of 16) of a row in a [128][128] tile with the 128-byte swizzle.
__device__ __forceinline__ uint32_t rt_at(int row, int ch) { return (ch >> 3) * kRtSub + row * 128 + (((ch & 7) ^ (row & 7)) << 4); }

__global__ void __launch_bounds__(kRtThreads, 1)
retention_chunk_kernel(const RetentionParams p, const float2* __restrict__ cs, float* __restrict__ o_raw, int row0, int N, int* status) {
  extern __shared__ uint8_t rt_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rt_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint8_t *q_sm = sm, *k_sm = q_sm + 2 * kRtTerm, *s_sm = k_sm + 2 * kRtTerm, *v_sm = s_sm + 2 * kRtTerm;
  float* pw = reinterpret_cast<float*>(v_sm + kRtTerm);    // decay^0 .. decay^128
  float* sums = pw + 132;                                  // [2][128]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sums + 256);
  uint64_t *bar_a = bars, *bar_o = bars + 1, *bar_s = bars + 2;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + 3);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = p.D, V = p.V, H = p.H, vtiles = (V + kRetTile - 1) / kRetTile;
  const int h = blockIdx.x / vtiles, v0 = (blockIdx.x - h * vtiles) * kRetTile, j = blockIdx.y, Vn = min(kRetTile, V - v0);
  if (warp == 0) {
    tmem_alloc(tmem_ptr, 512);
    tmem_relinquish();
  }
  if (tid == 32) {
    mbar_init(bar_a, 1), mbar_init(bar_o, 1), mbar_init(bar_s, 1);
    fence_mbar_init();
  }
  const float g = p.decay[h];
  if (tid < 129) pw[tid] = powf(g, static_cast<float>(tid));
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *tmem_ptr, T_A = tmem, T_Q = tmem + 128, T_O = tmem + 256, T_S = tmem + 384;
  pdl_trigger();
  pdl_wait();
  const int t0 = p.cu[j] - row0, t1 = p.cu[j + 1] - row0, slot = p.slots[j];
  const int q4 = warp & 3, half = warp >> 2, row = q4 * 32 + lane;      // TMEM lane (a query row, a value column) and half of the columns
  const uint32_t lanes = static_cast<uint32_t>(q4 * 32) << 16;
  float S[64];                                             // state of value column `row`, key channels 64 half .. + 63
  const bool fresh = slot < 0 || p.reset[j] != 0;
  float* mem = p.memory + (static_cast<size_t>(max(slot, 0)) * H + h) * D * V + v0 + row;
#pragma unroll
  for (int i = 0; i < 64; ++i) S[i] = !fresh && row < Vn && 64 * half + i < D ? mem[static_cast<size_t>(64 * half + i) * V] : 0.f;
  const auto stage_state = [&]() {
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      float f[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = S[8 * c + e];
      store_terms(s_sm + rt_at(row, 8 * half + c), f);
    }
  };
  stage_state();
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(p.proj) + static_cast<size_t>(row0) * p.ld;
  const __nv_bfloat16 *qp = proj + static_cast<size_t>(h) * D, *kp = proj + static_cast<size_t>(H + h) * D;
  const __nv_bfloat16 *vp = proj + 2ll * H * D + static_cast<size_t>(h) * V + v0, *gp = vp + static_cast<size_t>(H) * V;
  const float ks = rsqrtf(static_cast<float>(D));
  const int ch = tid & 15, r16 = tid >> 4, hc = p.rot / 16;             // staging: this thread's group of every row r16 + 16 n
  const int turn = ch < hc ? 1 : ch < 2 * hc ? 2 : 0, mate = (lane & 16) | (turn == 1 ? ch + hc : turn == 2 ? ch - hc : ch);
  const int DN = (D + 63) / 64 * 64, VN = (Vn + 63) / 64 * 64;
  const uint32_t id_a = umma_idesc_bf16(128, false, false), id_q = umma_idesc_bf16(VN, false, false), id_o = umma_idesc_bf16(VN, false, true),
                 id_s = umma_idesc_bf16(DN, true, true);
  uint32_t phase = 0;
  bool ok = true;
  for (int c0 = t0; c0 < t1; c0 += kRetTile, phase ^= 1u) {
    const int nt = min(kRetTile, t1 - c0);
    const bool has_state = !fresh || c0 > t0;
    // ---- the chunk's rows: rotated queries and keys as two terms, values; zero past the piece
#pragma unroll 1
    for (int n0 = 0; n0 < 8; n0 += 4) {
      uint4 qa[4], ka[4], va[4];
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int r = r16 + 16 * (n0 + n);
        const size_t at = static_cast<size_t>(c0 + r) * p.ld + ch * 8;
        const bool in = r < nt, dk = in && ch * 8 < D;
        qa[n] = dk ? *reinterpret_cast<const uint4*>(qp + at) : make_uint4(0, 0, 0, 0);
        ka[n] = dk ? *reinterpret_cast<const uint4*>(kp + at) : make_uint4(0, 0, 0, 0);
        va[n] = in && ch * 8 < Vn ? *reinterpret_cast<const uint4*>(vp + at) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int r = r16 + 16 * (n0 + n);
        float q[8], k[8];
        unpack8(qa[n], q);
        unpack8(ka[n], k);
        uint4 qm, km;                                      // the other half's values
        qm.x = __shfl_sync(0xffffffffu, qa[n].x, mate), qm.y = __shfl_sync(0xffffffffu, qa[n].y, mate);
        qm.z = __shfl_sync(0xffffffffu, qa[n].z, mate), qm.w = __shfl_sync(0xffffffffu, qa[n].w, mate);
        km.x = __shfl_sync(0xffffffffu, ka[n].x, mate), km.y = __shfl_sync(0xffffffffu, ka[n].y, mate);
        km.z = __shfl_sync(0xffffffffu, ka[n].z, mate), km.w = __shfl_sync(0xffffffffu, ka[n].w, mate);
        if (turn != 0 && r < nt) {
          float qo[8], ko[8];
          unpack8(qm, qo);
          unpack8(km, ko);
          const float2* a = cs + static_cast<size_t>(c0 + r) * (p.rot / 2) + (turn == 1 ? ch : ch - hc) * 8;
#pragma unroll
          for (int e = 0; e < 8; e += 2) {
            const float4 two = *reinterpret_cast<const float4*>(a + e);
            const float c1 = two.x, s1 = turn == 1 ? -two.y : two.y, c2 = two.z, s2 = turn == 1 ? -two.w : two.w;
            q[e] = fmaf(qo[e], s1, q[e] * c1), k[e] = fmaf(ko[e], s1, k[e] * c1);
            q[e + 1] = fmaf(qo[e + 1], s2, q[e + 1] * c2), k[e + 1] = fmaf(ko[e + 1], s2, k[e + 1] * c2);
          }
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) k[e] *= ks;
        const uint32_t at = rt_at(r, ch);
        store_terms(q_sm + at, q);
        store_terms(k_sm + at, k);
        *reinterpret_cast<uint4*>(v_sm + at) = va[n];
      }
    }
    fence_proxy_async_smem();
    tc_fence_before_sync();
    __syncthreads();
    const int kd = (D + 15) / 16, kt = (nt + 15) / 16;
    if (tid == 0) {
      tc_fence_after_sync();
      const uint32_t qa = smem_u32(q_sm), ka = smem_u32(k_sm), sa = smem_u32(s_sm);
      // terms: rounded x rounded, rounded x remainder, remainder x rounded
      for (int term = 0; term < 3; ++term) {
        const uint32_t a = qa + (term == 2 ? kRtTerm : 0), b = (term == 1 ? kRtTerm : 0);
        for (int kk = 0; kk < kd; ++kk) {
          const uint32_t off = (kk >> 2) * kRtSub + (kk & 3) * 32;
          const uint32_t acc = term > 0 || kk > 0 ? 1u : 0u;
          if (has_state) umma_bf16(T_Q, umma_desc_k_sw128(a + off), umma_desc_k_sw128(sa + b + off), id_q, acc);
          umma_bf16(T_A, umma_desc_k_sw128(a + off), umma_desc_k_sw128(ka + b + off), id_a, acc);
        }
      }
      umma_commit(bar_a);
    }
    __syncwarp();
    // the next chunk's rows and this one's gate come closer meanwhile
    for (int r = tid >> 1; r < kRetTile; r += kRtThreads / 2) {
      const int t = c0 + kRetTile + r;
      if (t < t1) {
        const __nv_bfloat16* src = (tid & 1) ? kp : qp;
        for (int c = 0; c < D; c += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(src + static_cast<size_t>(t) * p.ld + c));
        if (tid & 1)
          for (int c = 0; c < Vn; c += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(vp + static_cast<size_t>(t) * p.ld + c));
      }
      if ((tid & 1) == 0 && r < nt)
        for (int c = 0; c < Vn; c += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(gp + static_cast<size_t>(c0 + r) * p.ld + c));
    }
    ok = mbar_wait(bar_a, phase, status, kErrRetention);
    ok = __syncthreads_and(ok) != 0;
    if (!ok) break;
    tc_fence_after_sync();
    // ---- decayed scores in the queries' place; keys times their decay to the chunk's end
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      uint32_t a[32];
      tmem_ld_32x32(T_A + lanes + half * 64 + c * 32, a);
      tmem_ld_wait();
#pragma unroll
      for (int c8 = 0; c8 < 4; ++c8) {
        float f[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int col = half * 64 + c * 32 + c8 * 8 + e;
          f[e] = col <= row && col < nt ? __uint_as_float(a[c8 * 8 + e]) * pw[row - col] : 0.f;
        }
        store_terms(q_sm + rt_at(row, half * 8 + c * 4 + c8), f);
      }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int r = r16 + 16 * n;
      uint8_t* at = k_sm + rt_at(r, ch);
      float a[8], b[8];
      unpack8(*reinterpret_cast<const uint4*>(at), a);
      unpack8(*reinterpret_cast<const uint4*>(at + kRtTerm), b);
      const float w = r < nt ? pw[nt - 1 - r] : 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) a[e] = (a[e] + b[e]) * w;
      store_terms(at, a);
    }
    fence_proxy_async_smem();
    tc_fence_before_sync();
    __syncthreads();
    if (tid == 0) {
      tc_fence_after_sync();
      const uint32_t pa = smem_u32(q_sm), ka = smem_u32(k_sm), va = smem_u32(v_sm);
      for (int term = 0; term < 2; ++term)
        for (int kk = 0; kk < kt; ++kk)
          umma_bf16(T_O, umma_desc_k_sw128(pa + term * kRtTerm + (kk >> 2) * kRtSub + (kk & 3) * 32), umma_desc_mn_sw128(va + kk * 2048, kRtSub, 1024), id_o,
                    term > 0 || kk > 0 ? 1u : 0u);
      umma_commit(bar_o);
      for (int term = 0; term < 2; ++term)
        for (int kk = 0; kk < kt; ++kk)
          umma_bf16(T_S, umma_desc_mn_sw128(va + kk * 2048, kRtSub, 1024), umma_desc_mn_sw128(ka + term * kRtTerm + kk * 2048, kRtSub, 1024), id_s,
                    term > 0 || kk > 0 ? 1u : 0u);
      umma_commit(bar_s);
    }
    __syncwarp();
    // ---- rows: read-out and values together, norm, gate
    ok = mbar_wait(bar_o, phase, status, kErrRetention);
    tc_fence_after_sync();
    float o[64], ss = 0.f;
    const float lift = pw[min(row + 1, 128)];
    if (half * 64 < VN) {                                  // (the same for the whole warp)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t a[32];
        tmem_ld_32x32(T_O + lanes + half * 64 + c * 32, a);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) o[c * 32 + i] = __uint_as_float(a[i]);
        if (has_state) {
          tmem_ld_32x32(T_Q + lanes + half * 64 + c * 32, a);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[c * 32 + i] = fmaf(lift, __uint_as_float(a[i]), o[c * 32 + i]);
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) ss = fmaf(o[c * 32 + i], o[c * 32 + i], ss);
      }
    }
    sums[half * 128 + row] = ss;
    tc_fence_before_sync();
    ok = __syncthreads_and(ok) != 0;
    if (!ok) break;
    if (row < nt && half * 64 < VN) {
      const float rs = p.gain / sqrtf((sums[row] + sums[128 + row]) / V + p.norm_eps);
      const size_t t = static_cast<size_t>(c0 + row);
      const __nv_bfloat16* gate = gp + t * p.ld + half * 64;
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + (row0 + t) * p.ldo + static_cast<size_t>(h) * V + v0 + half * 64;
      float* raw = o_raw == nullptr ? nullptr : o_raw + (t * H + h) * ret_vp(V) + v0 + half * 64;
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        if (half * 64 + c * 8 < Vn) {
          if (raw != nullptr) {
            *reinterpret_cast<float4*>(raw + c * 8) = make_float4(o[c * 8], o[c * 8 + 1], o[c * 8 + 2], o[c * 8 + 3]);
            *reinterpret_cast<float4*>(raw + c * 8 + 4) = make_float4(o[c * 8 + 4], o[c * 8 + 5], o[c * 8 + 6], o[c * 8 + 7]);
          } else {
            float z[8];
            unpack8(*reinterpret_cast<const uint4*>(gate + c * 8), z);
#pragma unroll
            for (int e = 0; e < 8; ++e) z[e] = o[c * 8 + e] * rs * __fdividef(z[e], 1.f + __expf(fminf(-z[e], 80.f)));
            *reinterpret_cast<uint4*>(dst + c * 8) = make_uint4(pack_bf16(z[0], z[1]), pack_bf16(z[2], z[3]), pack_bf16(z[4], z[5]), pack_bf16(z[6], z[7]));
          }
        } else if (raw != nullptr && v0 + half * 64 + c * 8 < ret_vp(V)) {
          *reinterpret_cast<float4*>(raw + c * 8) = make_float4(0.f, 0.f, 0.f, 0.f);
          *reinterpret_cast<float4*>(raw + c * 8 + 4) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
      }
    }
    // ---- state
    ok = mbar_wait(bar_s, phase, status, kErrRetention);
    tc_fence_after_sync();
    const float fade = pw[nt];
    if (half * 64 < DN) {
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t a[32];
        tmem_ld_32x32(T_S + lanes + half * 64 + c * 32, a);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) S[c * 32 + i] = fmaf(fade, S[c * 32 + i], __uint_as_float(a[i]));
      }
    }
    if (c0 + kRetTile < t1) stage_state();
    tc_fence_before_sync();
    ok = __syncthreads_and(ok) != 0;
    if (!ok) break;
  }
  if (ok && slot >= 0 && t1 > t0) {
#pragma unroll
    for (int i = 0; i < 64; ++i)
      if (row < Vn && 64 * half + i < D) mem[static_cast<size_t>(64 * half + i) * V] = S[i];
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
}

// scratch: angles [N, rot / 2]; o_raw: rows of the unnormed result [N, H, ret_vp(V)] where a head is wider than a tile.
int launch_retention_chunks(const RetentionParams& p, float* scratch, float* o_raw, int pieces, int row0, int N, int* status, cudaStream_t st) {
  auto kern = retention_chunk_kernel;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kRtSmem);
    if (e != cudaSuccess) return static_cast<int>(e);
    prefer_max_shared(kern);
    configured = true;
  }
  auto* cs = reinterpret_cast<float2*>(scratch);
  const int half = p.rot / 2;
  if (half > 0) {
    const long long threads = static_cast<long long>(N) * half;
    if (threads > 0x7fffffffll) return -1;
    const int rc = static_cast<int>(launch_kernel(retention_angles_kernel, dim3(static_cast<unsigned>((threads + 255) / 256)), dim3(256), 0, st,
                                                  p.positions + row0, p.inv_freq, cs, half, N));
    if (rc) return rc;
  }
  const dim3 grid(p.H * ((p.V + kRetTile - 1) / kRetTile), pieces);
  return static_cast<int>(launch_kernel(kern, grid, dim3(kRtThreads), kRtSmem, st, p, cs, o_raw, row0, N, status));
}

}  // namespace mx
