// Retention of prompt portions in chunks on the 5th-generation tensor cores (tcgen05 + TMEM), bf16 rows.
//
// With decay g and the state S_0 before a chunk of n tokens (numbered from 0):
//   o_i = g^(i + 1) S_0^T q_i + sum_{j <= i} g^(i - j) (q_i . k_j) v_j          S_n = g^n S_0 + sum_j g^(n - 1 - j) k_j v_j^T
// A CTA owns one head (and 128 of its value columns) of one piece and walks its chunks of 128 tokens; per chunk four products:
//   scores   A = q k^T          read-out  Q = q S_0          values  O = (A masked by the decays) v          state  dS^T = v^T (decayed k)
// Everything that enters them is fp32 (rotated queries and keys, the state, decayed scores and keys) and is fed to the tensor
// cores as the sum of two bf16 terms (rounded value and remainder), the product of the two remainders left out: 16 bits of each
// operand, accumulated in fp32. The state itself stays in fp32 in tensor memory, where its product adds up, and is copied to shared memory
// as the next chunk's operand.
//
// The sixteen warps work in step: rotate and stage the chunk's rows, wait for scores and read-out, mask the scores (into the
// queries' place) and decay the keys (in place), wait for the values and finish the rows (norm, gate), wait for the state. Every
// wait is bounded and reports through the status word.
#include "api.h"
#include "retention.cuh"

namespace mx {

constexpr int kRtThreads = 512;
constexpr int kRtCols = 32;                                // columns of a [128][128] tile a thread takes of its row
constexpr int kRtSub = 128 * 128;                          // bytes of a [128 rows][64 columns] sub-tile
constexpr int kRtTerm = 2 * kRtSub;                        // bytes of a [128][128] bf16 tile
constexpr int kRtSmem = 1024 + 7 * kRtTerm + 2048;         // q, k, state as two terms each, v; decays, barriers
constexpr int kErrRetention = 501;
static_assert(kRtSmem <= 227 * 1024, "shared memory");

// Cosines of every token's angles [N, rot / 2], then the sines.
__global__ void __launch_bounds__(256)
retention_angles_kernel(const int* __restrict__ positions, const float* __restrict__ inv_freq, float* __restrict__ cs, int half, int N) {
  pdl_trigger();
  pdl_wait();
  const unsigned i = blockIdx.x * 256u + threadIdx.x, n = i / half;
  if (n >= static_cast<unsigned>(N)) return;
  float s, c;
  sincosf(static_cast<float>(positions[n]) * inv_freq[i - n * half], &s, &c);
  cs[i] = c;
  cs[static_cast<size_t>(N) * half + i] = s;
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

// Eight neighbouring values of a head, rotated, times a factor, as two terms. turn: 1 first half, 2 second half of the rotated
// dimensions, 0 neither; lane `mate` holds the other half's values (the whole warp comes here).
__device__ __forceinline__ void rotate_terms(const uint4& raw, int turn, int mate, const float (&c)[8], const float (&s)[8], float factor, uint8_t* hi) {
  uint4 m;
  m.x = __shfl_sync(0xffffffffu, raw.x, mate), m.y = __shfl_sync(0xffffffffu, raw.y, mate);
  m.z = __shfl_sync(0xffffffffu, raw.z, mate), m.w = __shfl_sync(0xffffffffu, raw.w, mate);
  float f[8], o[8];
  unpack8(raw, f);
  unpack8(m, o);
  const float sign = turn == 1 ? -1.f : 1.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) f[e] = (turn != 0 ? fmaf(sign * s[e], o[e], f[e] * c[e]) : f[e]) * factor;
  store_terms(hi, f);
}

__global__ void __launch_bounds__(kRtThreads, 1)
retention_chunk_kernel(const RetentionParams p, const float* __restrict__ cs, float* __restrict__ o_raw, int row0, int N, int* status) {
  extern __shared__ uint8_t rt_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rt_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint8_t *q_sm = sm, *k_sm = q_sm + 2 * kRtTerm, *s_sm = k_sm + 2 * kRtTerm, *v_sm = s_sm + 2 * kRtTerm;
  float* pw = reinterpret_cast<float*>(v_sm + kRtTerm);    // decay^0 .. decay^128
  float* sums = reinterpret_cast<float*>(s_sm);            // [4][128], between a chunk's read-out and the next state
  float* rows_sm = reinterpret_cast<float*>(q_sm);         // [128][128], once the decayed scores have been read
  uint64_t* bars = reinterpret_cast<uint64_t*>(pw + 132);
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
  const int q4 = warp & 3, col0 = (warp >> 2) * kRtCols, row = q4 * 32 + lane;   // TMEM lane (a query row, a value column), first column
  const uint32_t lanes = static_cast<uint32_t>(q4 * 32) << 16;
  const bool fresh = slot < 0 || p.reset[j] != 0;
  float* mem = p.memory + (static_cast<size_t>(max(slot, 0)) * H + h) * D * V + v0 + row;
  // a thread's part of the state (value column `row`, key channels from col0 on) as the next chunk's operand
  const auto stage_state = [&](const uint32_t (&a)[kRtCols]) {
#pragma unroll
    for (int c = 0; c < kRtCols / 8; ++c) {
      float f[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(a[8 * c + e]);
      store_terms(s_sm + rt_at(row, col0 / 8 + c), f);
    }
  };
  if (!fresh) {
    uint32_t a[kRtCols];
#pragma unroll
    for (int i = 0; i < kRtCols; ++i) a[i] = __float_as_uint(row < Vn && col0 + i < D ? mem[static_cast<size_t>(col0 + i) * V] : 0.f);
    tmem_st_32x32(T_S + lanes + col0, a);
    tmem_st_wait();
    stage_state(a);
  }
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(p.proj) + static_cast<size_t>(row0) * p.ld;
  const __nv_bfloat16 *qp = proj + static_cast<size_t>(h) * D, *kp = proj + static_cast<size_t>(H + h) * D;
  const __nv_bfloat16 *vp = proj + 2ll * H * D + static_cast<size_t>(h) * V + v0, *gp = vp + static_cast<size_t>(H) * V;
  const float ks = rsqrtf(static_cast<float>(D));
  constexpr int RS = kRtThreads / 16, RN = kRetTile / RS, RB = 2;       // staging: this thread's group of the rows r16 + RS n, RB at a time
  const int ch = tid & 15, r16 = tid >> 4, hc = p.rot / 16;
  const int turn = ch < hc ? 1 : ch < 2 * hc ? 2 : 0, mate = (lane & 16) | (turn == 1 ? ch + hc : turn == 2 ? ch - hc : ch);
  const float* angles = cs + (turn == 2 ? static_cast<size_t>(N) * (p.rot / 2) + (ch - hc) * 8 : static_cast<size_t>(ch) * 8);
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
    for (int n0 = 0; n0 < RN; n0 += RB) {
      uint4 qa[RB], ka[RB], va[RB];
      float4 ang[RB][2];
#pragma unroll
      for (int n = 0; n < RB; ++n) {
        const int r = r16 + RS * (n0 + n);
        const size_t at = static_cast<size_t>(c0 + r) * p.ld + ch * 8;
        const bool in = r < nt, dk = in && ch * 8 < D;
        qa[n] = dk ? *reinterpret_cast<const uint4*>(qp + at) : make_uint4(0, 0, 0, 0);
        ka[n] = dk ? *reinterpret_cast<const uint4*>(kp + at) : make_uint4(0, 0, 0, 0);
        va[n] = in && ch * 8 < Vn ? *reinterpret_cast<const uint4*>(vp + at) : make_uint4(0, 0, 0, 0);
        const float* a = angles + static_cast<size_t>(c0 + r) * (p.rot / 2);
        ang[n][0] = in && turn != 0 ? *reinterpret_cast<const float4*>(a) : make_float4(0.f, 0.f, 0.f, 0.f);
        ang[n][1] = in && turn != 0 ? *reinterpret_cast<const float4*>(a + 4) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int n = 0; n < RB; ++n) {
        const int r = r16 + RS * (n0 + n);
        const uint32_t at = rt_at(r, ch);
        float c[8], sn[8];                                 // a lane has loaded its half's cosines or sines, its mate the others
        const float mine[8] = {ang[n][0].x, ang[n][0].y, ang[n][0].z, ang[n][0].w, ang[n][1].x, ang[n][1].y, ang[n][1].z, ang[n][1].w};
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float other = __shfl_sync(0xffffffffu, mine[e], mate);
          c[e] = turn == 2 ? other : mine[e], sn[e] = turn == 2 ? mine[e] : other;
        }
        rotate_terms(qa[n], turn, mate, c, sn, 1.f, q_sm + at);
        rotate_terms(ka[n], turn, mate, c, sn, ks, k_sm + at);
        *reinterpret_cast<uint4*>(v_sm + at) = va[n];
      }
    }
    fence_proxy_async_smem();
    tc_fence_before_sync();
    __syncthreads();
    const int kd = (D + 15) / 16, kt = (nt + 15) / 16;
    if (tid == 0) {
      tc_fence_after_sync();
      const uint64_t qd = umma_desc_k_sw128(smem_u32(q_sm)), kds = umma_desc_k_sw128(smem_u32(k_sm)), sd = umma_desc_k_sw128(smem_u32(s_sm));
      constexpr uint64_t LOW = kRtTerm >> 4;               // (descriptors count 16-byte units)
      // terms: rounded x rounded, rounded x remainder, remainder x rounded
#pragma unroll
      for (int term = 0; term < 3; ++term) {
        const uint64_t a0 = qd + (term == 2 ? LOW : 0), b0 = kds + (term == 1 ? LOW : 0), c0d = sd + (term == 1 ? LOW : 0);
#pragma unroll
        for (int kk = 0; kk < 8; ++kk) {
          const uint64_t off = ((kk >> 2) * kRtSub + (kk & 3) * 32) >> 4;
          if (kk >= kd) break;
          if (has_state) umma_bf16(T_Q, a0 + off, c0d + off, id_q, term > 0 || kk > 0 ? 1u : 0u);
          umma_bf16(T_A, a0 + off, b0 + off, id_a, term > 0 || kk > 0 ? 1u : 0u);
        }
      }
      umma_commit(bar_a);
    }
    __syncwarp();
    // the next chunk's rows and this one's gates come closer meanwhile (not by the warp that issues: everybody waits for it)
    if (warp >= 8) {
      const int r = (tid >> 1) & 127, side = tid & 1;
      const auto closer = [](const __nv_bfloat16* src, int n) {
        for (int c = 0; c < n; c += 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(src + c));
      };
      const size_t at = static_cast<size_t>(c0 + r) * p.ld, next = at + static_cast<size_t>(kRetTile) * p.ld;
      if (side == 0 && o_raw == nullptr && r < nt) closer(gp + at, Vn);
      if (c0 + kRetTile + r < t1) {
        closer((side == 0 ? qp : kp) + next, D);
        if (side != 0) closer(vp + next, Vn);
      }
    }
    ok = mbar_wait(bar_a, phase, status, kErrRetention);
    ok = __syncthreads_and(ok) != 0;
    if (!ok) break;
    tc_fence_after_sync();
    // ---- decayed scores in the queries' place; keys times their decay to the chunk's end
    {
      uint32_t a[32];
      tmem_ld_32x32(T_A + lanes + col0, a);
      tmem_ld_wait();
#pragma unroll
      for (int c8 = 0; c8 < 4; ++c8) {
        float f[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int col = col0 + c8 * 8 + e;
          f[e] = col <= row && col < nt ? __uint_as_float(a[c8 * 8 + e]) * pw[row - col] : 0.f;
        }
        store_terms(q_sm + rt_at(row, col0 / 8 + c8), f);
      }
    }
    if (has_state && col0 < DN) {                          // the state fades over the chunk
      const float fade = pw[nt];
      uint32_t a[32];
      tmem_ld_32x32(T_S + lanes + col0, a);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; ++i) a[i] = __float_as_uint(__uint_as_float(a[i]) * fade);
      tmem_st_32x32(T_S + lanes + col0, a);
      tmem_st_wait();
    }
#pragma unroll
    for (int n = 0; n < RN; ++n) {
      const int r = r16 + RS * n;
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
      const uint64_t pd = umma_desc_k_sw128(smem_u32(q_sm)), vd = umma_desc_mn_sw128(smem_u32(v_sm), kRtSub, 1024),
                     wd = umma_desc_mn_sw128(smem_u32(k_sm), kRtSub, 1024);
      constexpr uint64_t LOW = kRtTerm >> 4, STEP = 2048 >> 4;
#pragma unroll
      for (int term = 0; term < 2; ++term)
#pragma unroll
        for (int kk = 0; kk < 8; ++kk) {
          if (kk >= kt) break;
          umma_bf16(T_O, pd + term * LOW + (((kk >> 2) * kRtSub + (kk & 3) * 32) >> 4), vd + kk * STEP, id_o, term > 0 || kk > 0 ? 1u : 0u);
        }
      umma_commit(bar_o);
#pragma unroll
      for (int term = 0; term < 2; ++term)
#pragma unroll
        for (int kk = 0; kk < 8; ++kk) {
          if (kk >= kt) break;
          umma_bf16(T_S, vd + kk * STEP, wd + term * LOW + kk * STEP, id_s, has_state || term > 0 || kk > 0 ? 1u : 0u);
        }
      umma_commit(bar_s);
    }
    __syncwarp();
    // ---- rows: read-out and values together, norm, gate
    uint4 gate[RN];
#pragma unroll
    for (int n = 0; n < RN; ++n) {
      const int r = r16 + RS * n;
      gate[n] = o_raw == nullptr && r < nt && ch * 8 < Vn ? *reinterpret_cast<const uint4*>(gp + static_cast<size_t>(c0 + r) * p.ld + ch * 8)
                                                          : make_uint4(0, 0, 0, 0);
    }
    ok = mbar_wait(bar_o, phase, status, kErrRetention);
    tc_fence_after_sync();
    float o[kRtCols], ss = 0.f;
    const float lift = pw[min(row + 1, 128)];
    if (col0 < VN) {                                       // (the same for the whole warp)
#pragma unroll
      for (int c = 0; c < kRtCols; c += 16) {
        uint32_t a[16];
        tmem_ld_32x16(T_O + lanes + col0 + c, a);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) o[c + i] = __uint_as_float(a[i]);
        if (has_state) {
          tmem_ld_32x16(T_Q + lanes + col0 + c, a);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[c + i] = fmaf(lift, __uint_as_float(a[i]), o[c + i]);
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) ss = fmaf(o[c + i], o[c + i], ss);
      }
    }
    sums[(col0 / kRtCols) * 128 + row] = ss;
    tc_fence_before_sync();
    ok = __syncthreads_and(ok) != 0;
    if (!ok) break;
    if (col0 < VN) {
      const float rs = o_raw != nullptr ? 1.f : p.gain / sqrtf(((sums[row] + sums[128 + row]) + (sums[256 + row] + sums[384 + row])) / V + p.norm_eps);
#pragma unroll
      for (int c = 0; c < kRtCols / 4; ++c)
        *reinterpret_cast<float4*>(rows_sm + row * kRetTile + 4 * ((col0 / 4 + c) ^ (row & 7))) =
            make_float4(o[4 * c] * rs, o[4 * c + 1] * rs, o[4 * c + 2] * rs, o[4 * c + 3] * rs);
    }
    __syncthreads();
#pragma unroll
    for (int n = 0; n < RN; ++n) {                         // whole rows go out together
      const int r = r16 + RS * n, col = ch * 8;
      if (r >= nt || v0 + col >= (o_raw != nullptr ? ret_vp(V) : V)) continue;
      const size_t t = static_cast<size_t>(c0 + r);
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;   // (columns past the head's are zero)
      if (col < Vn) {
        a = *reinterpret_cast<const float4*>(rows_sm + r * kRetTile + 4 * ((2 * ch) ^ (r & 7)));
        b = *reinterpret_cast<const float4*>(rows_sm + r * kRetTile + 4 * ((2 * ch + 1) ^ (r & 7)));
      }
      if (o_raw != nullptr) {
        float* raw = o_raw + (t * H + h) * ret_vp(V) + v0 + col;
        *reinterpret_cast<float4*>(raw) = a;
        *reinterpret_cast<float4*>(raw + 4) = b;
        continue;
      }
      float z[8];
      unpack8(gate[n], z);
      const float f[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
      for (int e = 0; e < 8; ++e) z[e] = f[e] * __fdividef(z[e], 1.f + __expf(fminf(-z[e], 80.f)));
      *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.out) + (row0 + t) * p.ldo + static_cast<size_t>(h) * V + v0 + col) =
          make_uint4(pack_bf16(z[0], z[1]), pack_bf16(z[2], z[3]), pack_bf16(z[4], z[5]), pack_bf16(z[6], z[7]));
    }
    // ---- state
    ok = mbar_wait(bar_s, phase, status, kErrRetention);
    tc_fence_after_sync();
    if (col0 < DN && ok) {
      uint32_t a[32];
      tmem_ld_32x32(T_S + lanes + col0, a);
      tmem_ld_wait();
      if (c0 + kRetTile < t1) {
        stage_state(a);
      } else if (slot >= 0) {
#pragma unroll
        for (int i = 0; i < kRtCols; ++i)
          if (row < Vn && col0 + i < D) mem[static_cast<size_t>(col0 + i) * V] = __uint_as_float(a[i]);
      }
    }
    tc_fence_before_sync();
    ok = __syncthreads_and(ok) != 0;
    if (!ok) break;
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
}

// scratch: cosines and sines of the angles [2, N, rot / 2]; o_raw: rows of the unnormed result [N, H, ret_vp(V)] where a head is wider than a tile.
int launch_retention_chunks(const RetentionParams& p, float* scratch, float* o_raw, int pieces, int row0, int N, int* status, cudaStream_t st) {
  auto kern = retention_chunk_kernel;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kRtSmem);
    if (e != cudaSuccess) return static_cast<int>(e);
    prefer_max_shared(kern);
    configured = true;
  }
  const int half = p.rot / 2;
  if (half > 0) {
    const long long threads = static_cast<long long>(N) * half;
    if (threads > 0x7fffffffll) return -1;
    const int rc = static_cast<int>(launch_kernel(retention_angles_kernel, dim3(static_cast<unsigned>((threads + 255) / 256)), dim3(256), 0, st,
                                                  p.positions + row0, p.inv_freq, scratch, half, N));
    if (rc) return rc;
  }
  const dim3 grid(p.H * ((p.V + kRetTile - 1) / kRetTile), pieces);
  return static_cast<int>(launch_kernel(kern, grid, dim3(kRtThreads), kRtSmem, st, p, scratch, o_raw, row0, N, status));
}

}  // namespace mx
