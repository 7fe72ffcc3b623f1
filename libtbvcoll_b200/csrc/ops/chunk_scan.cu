// chunk_scan.cu — the recurrence of decay_scan.cu for many rows of a bf16 model, in chunks of 16 tokens on tensor cores.
//
// With P_t the product of the decays from the chunk's first token to t (per key channel; for WKV to t - 1), R_s the product after s to its last, and
// S the state before the chunk:
//   o_t = (q_t P_t)^T S + sum_{s <= t} A_ts v_s          A_ts = sum_d q_t k_s * (product of the decays between s and t)
//   S  <- diag(P_16) S + sum_s (k_s R_s) v_s^T
// Every factor is a running product of decays, at most 1: nothing is divided and no exponent can overflow, however strong the decay.  A's two
// triangles of 8 x 8 come from running products in registers, its remaining 8 x 8 block is a product of rows scaled to the middle of the chunk.
//
// S^T lives in the accumulators of the warps: warp w owns 16 value columns x all key channels.  As accumulator layout equals operand layout, it is
// also the left operand of the readout.  v is bf16 as it stands.  fp32 operands are carried as sums of bf16 numbers: k_s R_s as three (24 bits: the
// state is updated as in fp32), q_t P_t, S and A as two for the readout, whose result is rounded to bf16 behind the head norm.
//
// The decay inputs come from memory (p.z) or from the low-rank product itself: z = low . w2^T + b2 for a chunk is a few products per warp with w2's
// rows of the head in shared memory.  If a CTA owns all value columns of its head, head norm, weight and gate follow here as well.
//
// A CTA alternates between making a chunk's operands (elementwise, shared memory) and its products; two CTAs per SM overlap the two.
// Long segments are cut into groups that run in parallel: states of all groups but a segment's last from zero (k_chunk_scan<true>), then the
// states they start from (k_group_starts), then all outputs.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../pdl.cuh"
#include "attn_mma.cuh"
#include "decay.cuh"
#include "vec.cuh"

using namespace attn_mma;
using decay_ops::decay;
using decay_ops::ScanParams;

namespace {

constexpr int kC = 16;

template <int DK>
struct Shape {
  static constexpr int kItemWarps = DK / 16;                       // 16 channels x 2 halves of the chunk each
  static constexpr int NI = kItemWarps > 8 ? 2 : 1;                // items per warp
  static constexpr int NW = kItemWarps / NI;                       // warps of a CTA; each owns 16 value columns
  static constexpr int kPitch = DK * 2 + 16;                       // bytes; odd multiple of 16: ldmatrix without conflicts
  static constexpr int kVPitch = NW * 32 + 16;
  static constexpr int kAPitch = kC * 2 + 16;
  // byte offsets of dynamic shared memory
  static constexpr int oQ = 0;                                     // q P: hi, lo         [2][16][pitch]
  static constexpr int oK = oQ + 2 * kC * kPitch;                  // k R: hi, mid, lo    [3][16][pitch]
  static constexpr int oQm = oK + 3 * kC * kPitch;                 // second half, from the middle: hi, lo  [2][8][pitch]
  static constexpr int oKm = oQm + 2 * 8 * kPitch;                 // first half, to the middle             [2][8][pitch]
  static constexpr int oV = oKm + 2 * 8 * kPitch;                  // v                   [2 chunks][16][vpitch]
  static constexpr int oA = oV + 2 * kC * kVPitch;                 // A: hi, lo           [2][16][apitch]
  static constexpr int oZ = oA + 2 * kC * kAPitch;                 // raw decay inputs    [16][DK] fp32
  static constexpr int oRq = oZ + kC * DK * 4;                     // raw q, k            [16][DK] bf16 each
  static constexpr int oRk = oRq + kC * DK * 2;
  static constexpr int oE = oRk + kC * DK * 2;                     // P_16                [DK] fp32
  static constexpr int oTri = oE + DK * 4;                         // triangles           [2 chunks][item warps][2][36] fp32
  static constexpr int oOff = oTri + 2 * kItemWarps * 72 * 4;      // the block between the halves [warps][64] fp32
  static constexpr int kOPitch = NW * 16 + 4;                      // floats
  static constexpr int oO = oOff + NW * 64 * 4;                    // o                   [16][opitch] fp32
  static constexpr int oG = oO + kC * kOPitch * 4;                 // gates               [16][vpitch] bf16
  static constexpr int oLow = oG + kC * kVPitch;                   // low                 [2 chunks][16][rank pitch], then w2 [DK][rank pitch]
  static constexpr int bytes(int rank) { return oLow + (rank ? (2 * kC + DK) * (rank * 2 + 16) : 0); }
};

__device__ __forceinline__ float bf16_to_f(uint32_t bits) { return __uint_as_float(bits << 16); }
// x = hi + lo (+ lo2), bf16 each; stored at the given shared addresses
__device__ __forceinline__ void st_bf16(uint32_t addr, __nv_bfloat16 v) { asm volatile("st.shared.b16 [%0], %1;" ::"r"(addr), "h"(*reinterpret_cast<unsigned short*>(&v)) : "memory"); }
__device__ __forceinline__ void split2(float x, uint32_t hi, uint32_t lo) {
  const __nv_bfloat16 h = __float2bfloat16_rn(x);
  st_bf16(hi, h);
  st_bf16(lo, __float2bfloat16_rn(x - __bfloat162float(h)));
}
__device__ __forceinline__ void split3(float x, uint32_t hi, uint32_t mid, uint32_t lo) {
  const __nv_bfloat16 h = __float2bfloat16_rn(x);
  const float r = x - __bfloat162float(h);
  const __nv_bfloat16 m = __float2bfloat16_rn(r);
  st_bf16(hi, h);
  st_bf16(mid, m);
  st_bf16(lo, __float2bfloat16_rn(r - __bfloat162float(m)));
}
__device__ __forceinline__ void pack_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

template <int DK, bool STATE_ONLY, bool LOW>
__global__ void __launch_bounds__(Shape<DK>::NW * 32, DK > 128 ? 1 : (DK > 64 ? 2 : 3)) k_chunk_scan(const ScanParams p, const int* groups, float* starts, float* totals) {
  using S = Shape<DK>;
  constexpr int NW = S::NW, NI = S::NI, NT = NW * 32;
  extern __shared__ __align__(16) uint8_t sm[];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r8 = lane >> 2, quad = lane & 3;
  const int h = blockIdx.y, gi = blockIdx.x;
  const int first = groups[4 * gi], n = groups[4 * gi + 1], slot = groups[4 * gi + 2], flags = groups[4 * gi + 3];
  if (STATE_ONLY && !(flags & 2)) return;
  const bool wkv = p.u != nullptr, fresh = p.positions[first] == 0;
  const int vb = blockIdx.z * NW * 16, v0 = vb + warp * 16;         // first value column of the CTA, of the warp
  const bool mma_warp = v0 < p.Vp;
  const uint32_t base = smem_addr(sm);
  const size_t hs = size_t(p.Dp) * p.Vp;                            // state values per head
  const __nv_bfloat16* qg = static_cast<const __nv_bfloat16*>(p.q) + size_t(h) * p.Dp;
  const __nv_bfloat16* kg = static_cast<const __nv_bfloat16*>(p.k) + size_t(h) * p.Dp;
  const __nv_bfloat16* vg = static_cast<const __nv_bfloat16*>(p.v) + size_t(h) * p.Vp + vb;
  const float* zg = p.z + size_t(h) * p.Dp;

  // rows of chunk c on their way to shared memory; missing rows of v are zeros, the others' are left out when they are used
  auto issue = [&](int c) {
    const int at = c * kC, nt = min(kC, n - at), dch = p.Dp / 8, vch = min(NW * 16, p.Vp - vb) / 8;
    if (!LOW) for (int i = tid; i < nt * dch * 2; i += NT) {
      const int t = i / (dch * 2), x = i - t * dch * 2;
      cp_async16(base + S::oZ + (t * DK + x * 4) * 4, zg + size_t(first + at + t) * p.ldz + x * 4);
    }
    for (int i = tid; i < nt * dch; i += NT) {
      const int t = i / dch, x = i - t * dch;
      if (!STATE_ONLY) cp_async16(base + S::oRq + (t * DK + x * 8) * 2, qg + size_t(first + at + t) * p.ld + x * 8);
      cp_async16(base + S::oRk + (t * DK + x * 8) * 2, kg + size_t(first + at + t) * p.ld + x * 8);
    }
    const uint32_t vbuf = base + S::oV + (c & 1) * kC * S::kVPitch;
    for (int i = tid; i < kC * vch; i += NT) {
      const int t = i / vch, x = i - t * vch;
      if (t < nt) cp_async16(vbuf + t * S::kVPitch + x * 16, vg + size_t(first + at + t) * p.ld + x * 8);
      else st_zero16(vbuf + t * S::kVPitch + x * 16);
    }
  };
  const int lpitch = p.rank * 2 + 16;
  const uint32_t w2s = base + S::oLow + 2 * kC * lpitch;
  auto issue_low = [&](int c) {
    const int at = c * kC, nt = min(kC, n - at), ch = p.rank / 8;
    for (int i = tid; i < nt * ch; i += NT) {
      const int t = i / ch, x = i - t * ch;
      cp_async16(base + S::oLow + ((c & 1) * kC + t) * lpitch + x * 16, static_cast<const __nv_bfloat16*>(p.low) + size_t(first + at + t) * p.ldlow + x * 8);
    }
  };
  // decay inputs of chunk c: tokens x channels, 16 channels per warp and item
  auto decay_product = [&](int c) {
#pragma unroll
    for (int it = 0; it < NI; it++) {
      const int d0 = (warp + it * NW) * 16;
      float acc[2][4] = {};
      for (int ks = 0; ks < p.rank / 16; ks++) {
        uint32_t a[4], b[4];
        ldmatrix_x4(base + S::oLow + ((c & 1) * kC + (lane & 15)) * lpitch + (lane >> 4) * 16 + ks * 32, a);
        ldmatrix_x4(w2s + (d0 + (lane & 7) + ((lane >> 4) << 3)) * lpitch + ((lane >> 3) & 1) * 16 + ks * 32, b);
        mma_bf16(acc[0], a, b[0], b[1]);
        mma_bf16(acc[1], a, b[2], b[3]);
      }
#pragma unroll
      for (int i = 0; i < 2; i++) {
        const int d = d0 + i * 8 + quad * 2;
        float2 b = make_float2(0.f, 0.f);
        if (d < p.Dp) b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(static_cast<const __nv_bfloat16*>(p.b2) + size_t(h) * p.Dp + d));
        float* z = reinterpret_cast<float*>(sm + S::oZ) + r8 * DK + d;
        *reinterpret_cast<float2*>(z) = make_float2(acc[i][0] + b.x, acc[i][1] + b.y);
        *reinterpret_cast<float2*>(z + 8 * DK) = make_float2(acc[i][2] + b.x, acc[i][3] + b.y);
      }
    }
  };
  // head norm, weight and gate of chunk c, whose o lies in shared memory; a row per 2 NW lanes, 8 columns per lane
  const bool fused = !STATE_ONLY && p.o == nullptr;
  auto issue_gates = [&](int c) {
    const int at = c * kC, nt = min(kC, n - at), vch = p.Vp / 8;
    for (int i = tid; i < nt * vch; i += NT) {
      const int t = i / vch, x = i - t * vch;
      cp_async16(base + S::oG + t * S::kVPitch + x * 16, static_cast<const __nv_bfloat16*>(p.g) + size_t(first + at + t) * p.ld + size_t(h) * p.Vp + x * 8);
    }
  };
  auto emit = [&](int c) {
    const int t = tid / (2 * NW), v = tid % (2 * NW) * 8;
    float f[8], ss = 0.f;
    vec::load8(reinterpret_cast<const float*>(sm + S::oO) + t * S::kOPitch + v, f);
    if (v >= p.Vp) {
#pragma unroll
      for (int e = 0; e < 8; e++) f[e] = 0.f;
    }
#pragma unroll
    for (int e = 0; e < 8; e++) ss = fmaf(f[e], f[e], ss);
#pragma unroll
    for (int o = NW; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (c * kC + t < n && v < p.Vp) {
      const float r = 1.0f / sqrtf(ss / float(p.vdim) + p.eps);
      float g[8], w[8];
      vec::load8(reinterpret_cast<const __nv_bfloat16*>(sm + S::oG + t * S::kVPitch) + v, g);
      vec::load8(p.norm + size_t(h) * p.Vp + v, w);
#pragma unroll
      for (int e = 0; e < 8; e++) f[e] = f[e] * r * w[e] * vec::gate<__nv_bfloat16>(g[e]);
      vec::store8(static_cast<__nv_bfloat16*>(p.out) + size_t(first + c * kC + t) * p.ldo + size_t(h) * p.Vp + v, f);
    }
  };

  float etot[NI];
#pragma unroll
  for (int i = 0; i < NI; i++) etot[i] = 1.f;

  // operands of chunk c
  auto prepare = [&](int c) {
    const int nt = min(kC, n - c * kC);
#pragma unroll
    for (int it = 0; it < NI; it++) {
      const int iw = warp + it * NW, d = iw * 16 + (lane & 15), half = lane >> 4;
      const bool in = d < p.Dp;
      float a[8], q[8], k[8];
#pragma unroll
      for (int j = 0; j < 8; j++) {
        const int t = half * 8 + j;
        const bool ok = in && t < nt;
        const float z = *reinterpret_cast<const float*>(sm + S::oZ + (t * DK + d) * 4);
        a[j] = ok ? decay<__nv_bfloat16>(z, wkv, p.inv_tau) : 1.f;
        k[j] = ok ? __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(sm + S::oRk + (t * DK + d) * 2)) : 0.f;
        if (!STATE_ONLY) q[j] = ok ? __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(sm + S::oRq + (t * DK + d) * 2)) * p.qscale : 0.f;
      }
      float tot = 1.f;
#pragma unroll
      for (int j = 0; j < 8; j++) tot *= a[j];
      const float other = __shfl_xor_sync(0xffffffffu, tot, 16);
      if (half == 0) {
        *reinterpret_cast<float*>(sm + S::oE + d * 4) = tot * other;
        etot[it] *= tot * other;
      }
      // k R: running products from the end
      const float beyond = half == 0 ? other : 1.f;
      float run = 1.f;
#pragma unroll
      for (int j = 7; j >= 0; j--) {
        const float km = k[j] * run;
        const uint32_t at = base + S::oK + (half * 8 + j) * S::kPitch + d * 2;
        split3(km * beyond, at, at + kC * S::kPitch, at + 2 * kC * S::kPitch);
        if (!STATE_ONLY && half == 0) split2(km, base + S::oKm + j * S::kPitch + d * 2, base + S::oKm + (8 + j) * S::kPitch + d * 2);
        run *= a[j];
      }
      if (STATE_ONLY) continue;
      // q P: running products from the start, the current token's decay included (not for WKV)
      const float before = half == 1 ? other : 1.f;
      run = 1.f;
#pragma unroll
      for (int j = 0; j < 8; j++) {
        if (!wkv) run *= a[j];
        const float qm = q[j] * run;
        const uint32_t at = base + S::oQ + (half * 8 + j) * S::kPitch + d * 2;
        split2(qm * before, at, at + kC * S::kPitch);
        if (half == 1) split2(qm, base + S::oQm + j * S::kPitch + d * 2, base + S::oQm + (8 + j) * S::kPitch + d * 2);
        if (wkv) run *= a[j];
      }
      // the triangle of this half: values (t, s <= t) in row order, eight at a time summed over the 16 channels of the half-warp
      const float u = wkv && in ? p.u[size_t(h) * p.Dp + d] : 1.f;
      float* tri = reinterpret_cast<float*>(sm + S::oTri) + (((c & 1) * S::kItemWarps + iw) * 2 + half) * 36;
      float val[8];
      int w = 0;
#pragma unroll
      for (int t = 0; t < 8; t++) {
        // k[s], s < t, holds k_s times the decays between s and t
        if (!wkv) {
#pragma unroll
          for (int s = 0; s < t; s++) k[s] *= a[t];
        }
#pragma unroll
        for (int s = 0; s <= t; s++) {
          val[w & 7] = q[t] * k[s] * (s == t ? u : 1.f);
          w++;
          if ((w & 7) == 0 || w == 36) {
            const int cnt = w == 36 ? 4 : 8, p0 = w - cnt;
            int idx = 0;
            if (cnt == 8) {
#pragma unroll
              for (int j = 0; j < 4; j++) {
                const float send = lane & 8 ? val[j] : val[j + 4], keep = lane & 8 ? val[j + 4] : val[j];
                val[j] = keep + __shfl_xor_sync(0xffffffffu, send, 8);
              }
              idx += lane & 8 ? 4 : 0;
            } else {
#pragma unroll
              for (int j = 0; j < 4; j++) val[j] += __shfl_xor_sync(0xffffffffu, val[j], 8);
            }
#pragma unroll
            for (int j = 0; j < 2; j++) {
              const float send = lane & 4 ? val[j] : val[j + 2], keep = lane & 4 ? val[j + 2] : val[j];
              val[j] = keep + __shfl_xor_sync(0xffffffffu, send, 4);
            }
            idx += lane & 4 ? 2 : 0;
            const float send = lane & 2 ? val[0] : val[1], keep = lane & 2 ? val[1] : val[0];
            float sum = keep + __shfl_xor_sync(0xffffffffu, send, 2);
            idx += lane & 2 ? 1 : 0;
            sum += __shfl_xor_sync(0xffffffffu, sum, 1);
            if ((lane & 1) == 0) tri[p0 + idx] = sum;
          }
        }
        if (wkv) {
#pragma unroll
          for (int s = 0; s < t; s++) k[s] *= a[t];
        }
      }
    }
  };
  // A of chunk c from its pieces
  auto assemble = [&](int c) {
    const float* tri = reinterpret_cast<const float*>(sm + S::oTri) + (c & 1) * S::kItemWarps * 72;
    const float* off = reinterpret_cast<const float*>(sm + S::oOff);
    for (int e = tid; e < kC * kC; e += NT) {
      const int t = e >> 4, s = e & 15;
      float v = 0.f;
      if (s <= t) {
        if ((t ^ s) & 8) {
#pragma unroll
          for (int w = 0; w < NW; w++) v += off[w * 64 + (t & 7) * 8 + s];
        } else {
          const int tt = t & 7, ss = s & 7, at = (t >> 3) * 36 + tt * (tt + 1) / 2 + ss;
#pragma unroll
          for (int w = 0; w < S::kItemWarps; w++) v += tri[w * 72 + at];
        }
      }
      const uint32_t at = base + S::oA + t * S::kAPitch + s * 2;
      split2(v, at, at + kC * S::kAPitch);
    }
  };

  float st[DK / 8][4];      // S^T: value column v0 + r8 (+ 8), channels 8 i + 2 quad (+ 1)
  const bool multi = flags != 0;
  const float* from = multi ? starts + (size_t(gi) * p.heads + h) * hs : p.state + (size_t(slot) * p.heads + h) * hs;
  const bool zero = STATE_ONLY || !mma_warp || (!multi && fresh);
#pragma unroll
  for (int i = 0; i < DK / 8; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int d = i * 8 + quad * 2 + (j & 1), v = v0 + r8 + (j >> 1) * 8;
      st[i][j] = zero || d >= p.Dp ? 0.f : from[size_t(d) * p.Vp + v];
    }

  float o[2][4];            // o^T: value column as above, tokens 8 i + 2 quad (+ 1)
  uint32_t vf[4];           // v^T of the current chunk
  const uint32_t brow = (lane & 7) + ((lane >> 4) << 3), bcol = ((lane >> 3) & 1) * 16;    // right operands stored [n][k]
  auto finish = [&](int c) {
    // adds A v, stores the outputs
    uint32_t b[4];
#pragma unroll
    for (int x = 0; x < 2; x++) {
      ldmatrix_x4(base + S::oA + x * kC * S::kAPitch + brow * S::kAPitch + bcol, b);
      mma_bf16(o[0], vf, b[0], b[1]);
      mma_bf16(o[1], vf, b[2], b[3]);
    }
    const int at = c * kC;
#pragma unroll
    for (int i = 0; i < 2; i++)
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const int t = i * 8 + quad * 2 + (j & 1), v = r8 + (j >> 1) * 8;
        if (fused) reinterpret_cast<float*>(sm + S::oO)[t * S::kOPitch + warp * 16 + v] = o[i][j];
        else if (at + t < n) p.o[(size_t(first + at + t) * p.heads + h) * p.Vp + v0 + v] = o[i][j];
      }
  };

  const int nc = (n + kC - 1) / kC;
  if (LOW) {
    const int ch = p.rank / 8;
    for (int i = tid; i < p.Dp * ch; i += NT) {
      const int d = i / ch, x = i - d * ch;
      cp_async16(w2s + d * lpitch + x * 16, static_cast<const __nv_bfloat16*>(p.w2) + (size_t(h) * p.Dp + d) * p.rank + x * 8);
    }
    issue_low(0);
    if (nc > 1) issue_low(1);
  }
  issue(0);
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  if (LOW) {
    decay_product(0);
    __syncthreads();
  }
  prepare(0);
  __syncthreads();
  for (int c = 0; c < nc; c++) {
    if (c + 1 < nc) issue(c + 1);
    if (LOW && c + 2 < nc) issue_low(c + 2);
    if (fused && c > 0) issue_gates(c - 1);
    cp_async_commit();
    if (LOW && c + 1 < nc) decay_product(c + 1);
    if (mma_warp) {
      if (!STATE_ONLY) {
        if (c > 0) finish(c - 1);
#pragma unroll
        for (int i = 0; i < 2; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DK / 16; ks++) {
          uint32_t sh[4], sl[4], bh[4], bl[4];
          ldmatrix_x4(base + S::oQ + brow * S::kPitch + bcol + ks * 32, bh);
          ldmatrix_x4(base + S::oQ + kC * S::kPitch + brow * S::kPitch + bcol + ks * 32, bl);
          pack_split(st[2 * ks][0], st[2 * ks][1], sh[0], sl[0]);
          pack_split(st[2 * ks][2], st[2 * ks][3], sh[1], sl[1]);
          pack_split(st[2 * ks + 1][0], st[2 * ks + 1][1], sh[2], sl[2]);
          pack_split(st[2 * ks + 1][2], st[2 * ks + 1][3], sh[3], sl[3]);
          mma_bf16(o[0], sh, bh[0], bh[1]);
          mma_bf16(o[1], sh, bh[2], bh[3]);
          mma_bf16(o[0], sh, bl[0], bl[1]);
          mma_bf16(o[1], sh, bl[2], bl[3]);
          mma_bf16(o[0], sl, bh[0], bh[1]);
          mma_bf16(o[1], sl, bh[2], bh[3]);
        }
      }
      // v^T: stored [token][column]
      ldmatrix_x4_trans(base + S::oV + (c & 1) * kC * S::kVPitch + ((lane & 7) + ((lane >> 4) << 3)) * S::kVPitch + (warp * 16 + ((lane >> 3) & 1) * 8) * 2, vf);
#pragma unroll
      for (int i = 0; i < DK / 8; i++) {
        const float2 e = *reinterpret_cast<const float2*>(sm + S::oE + (i * 8 + quad * 2) * 4);
        st[i][0] *= e.x; st[i][1] *= e.y; st[i][2] *= e.x; st[i][3] *= e.y;
      }
#pragma unroll
      for (int i = 0; i < DK / 16; i++) {
#pragma unroll
        for (int x = 2; x >= 0; x--) {            // smallest part first
          uint32_t b[4];
          ldmatrix_x4_trans(base + S::oK + x * kC * S::kPitch + (lane & 15) * S::kPitch + i * 32 + (lane >> 4) * 16, b);
          mma_bf16(st[2 * i], vf, b[0], b[1]);
          mma_bf16(st[2 * i + 1], vf, b[2], b[3]);
        }
      }
    }
    if (!STATE_ONLY) {
      // the block between the halves: second-half rows against first-half rows, k steps shared out over the warps
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      for (int ks = warp; ks < DK / 16; ks += NW) {
        const uint32_t row = (lane & 7) * S::kPitch + ((lane >> 3) & 1) * 16 + ks * 32;
        uint32_t ah[4] = {0, 0, 0, 0}, al[4] = {0, 0, 0, 0}, bh[2], bl[2], x[2];
        ldmatrix_x2(base + S::oQm + row, x);
        ah[0] = x[0]; ah[2] = x[1];
        ldmatrix_x2(base + S::oQm + 8 * S::kPitch + row, x);
        al[0] = x[0]; al[2] = x[1];
        ldmatrix_x2(base + S::oKm + row, bh);
        ldmatrix_x2(base + S::oKm + 8 * S::kPitch + row, bl);
        mma_bf16(acc, ah, bl[0], bl[1]);
        mma_bf16(acc, al, bh[0], bh[1]);
        mma_bf16(acc, ah, bh[0], bh[1]);
      }
      *reinterpret_cast<float2*>(sm + S::oOff + (warp * 64 + r8 * 8 + quad * 2) * 4) = make_float2(acc[0], acc[1]);
    }
    cp_async_wait<0>();
    __syncthreads();
    if (!STATE_ONLY) assemble(c);
    if (fused && c > 0) emit(c - 1);
    if (c + 1 < nc) prepare(c + 1);
    __syncthreads();
  }
  if (fused) {
    issue_gates(nc - 1);
    cp_async_commit();
  }
  if (mma_warp && !STATE_ONLY) finish(nc - 1);
  if (fused) {
    cp_async_wait<0>();
    __syncthreads();
    emit(nc - 1);
  }
  if (mma_warp) {
    float* to = STATE_ONLY ? starts + (size_t(gi + 1) * p.heads + h) * hs : p.state + (size_t(slot) * p.heads + h) * hs;
    if (STATE_ONLY || !(flags & 2)) {
#pragma unroll
      for (int i = 0; i < DK / 8; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
          const int d = i * 8 + quad * 2 + (j & 1), v = v0 + r8 + (j >> 1) * 8;
          if (d < p.Dp) to[size_t(d) * p.Vp + v] = st[i][j];
        }
    }
  }
  if (STATE_ONLY) {
    if (blockIdx.z == 0) {
#pragma unroll
      for (int it = 0; it < NI; it++) {
        const int d = (warp + it * NW) * 16 + (lane & 15);
        if (lane < 16 && d < p.Dp) totals[(size_t(gi) * p.heads + h) * p.Dp + d] = etot[it];
      }
    }
  } else if (p.h1 && !(flags & 2)) {
    const int ctas = gridDim.y * gridDim.z, id = blockIdx.z * gridDim.y + blockIdx.y;
    for (int i = id * NT + tid; i < p.ldh; i += ctas * NT) p.shift[size_t(slot) * p.ldh + i] = p.h1[size_t(first + n - 1) * p.ldh + i];
  }
}

// Before: starts[g + 1] = the state that group g alone leaves (from zero), totals[g] = its decays' products.  After: starts[g] = the state that
// group g starts from.  One CTA column per segment of several groups (at its first group).
__global__ void __launch_bounds__(256) k_group_starts(const ScanParams p, const int* groups, float* starts, const float* totals) {
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  int g = blockIdx.x;
  const int h = blockIdx.y, i = blockIdx.z * 256 + threadIdx.x, hv = p.Dp * p.Vp / 4;
  if (groups[4 * g + 3] != 2 || i >= hv) return;
  const int d = i * 4 / p.Vp;
  const bool fresh = p.positions[groups[4 * g]] == 0;
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (!fresh) s = reinterpret_cast<const float4*>(p.state)[(size_t(groups[4 * g + 2]) * p.heads + h) * hv + i];
  float4* at = reinterpret_cast<float4*>(starts) + (size_t(g) * p.heads + h) * hv + i;
  *at = s;
  while (groups[4 * g + 3] & 2) {
    const float e = totals[(size_t(g) * p.heads + h) * p.Dp + d];
    g++;
    at += size_t(p.heads) * hv;
    const float4 l = *at;
    s = make_float4(fmaf(e, s.x, l.x), fmaf(e, s.y, l.y), fmaf(e, s.z, l.z), fmaf(e, s.w, l.w));
    *at = s;
  }
}

template <int DK, bool STATE_ONLY, bool LOW>
cudaError_t launch(const ScanParams& p, const int* groups, int ngroups, float* starts, float* totals, cudaStream_t st) {
  using S = Shape<DK>;
  static bool done = false;
  const size_t smem = size_t(S::bytes(LOW ? p.rank : 0));
  cudaError_t e = allow_smem(k_chunk_scan<DK, STATE_ONLY, LOW>, smem, &done);
  return e != cudaSuccess ? e : pdl::launch(k_chunk_scan<DK, STATE_ONLY, LOW>, dim3(ngroups, p.heads, (p.Vp / 16 + S::NW - 1) / S::NW), dim3(S::NW * 32), smem, st, 1, p,
                                            groups, starts, totals);
}
template <int DK, bool LOW>
cudaError_t run(ScanParams p, const int* groups, int ngroups, bool multi, float* starts, float* totals, bool* finished, cudaStream_t st) {
  *finished = p.Vp <= Shape<DK>::NW * 16;
  if (*finished) p.o = nullptr;
  cudaError_t e = cudaSuccess;
  if (multi) {
    e = launch<DK, true, LOW>(p, groups, ngroups, starts, totals, st);
    if (e == cudaSuccess) e = pdl::launch(k_group_starts, dim3(ngroups, p.heads, (p.Dp * p.Vp / 4 + 255) / 256), dim3(256), 0, st, 1, p, groups, starts, static_cast<const float*>(totals));
  }
  return e != cudaSuccess ? e : launch<DK, false, LOW>(p, groups, ngroups, starts, totals, st);
}
template <int DK>
cudaError_t run(const ScanParams& p, const int* groups, int ngroups, bool multi, float* starts, float* totals, bool* finished, cudaStream_t st) {
  return p.z ? run<DK, false>(p, groups, ngroups, multi, starts, totals, finished, st) : run<DK, true>(p, groups, ngroups, multi, starts, totals, finished, st);
}

}  // namespace

namespace decay_ops {

cudaError_t chunk_scan(const ScanParams& p, const int* groups, int ngroups, bool multi, float* starts, float* totals, bool* finished, cudaStream_t st) {
  if (p.Dp <= 32) return run<32>(p, groups, ngroups, multi, starts, totals, finished, st);
  if (p.Dp <= 64) return run<64>(p, groups, ngroups, multi, starts, totals, finished, st);
  if (p.Dp <= 128) return run<128>(p, groups, ngroups, multi, starts, totals, finished, st);
  return run<256>(p, groups, ngroups, multi, starts, totals, finished, st);
}

}  // namespace decay_ops
