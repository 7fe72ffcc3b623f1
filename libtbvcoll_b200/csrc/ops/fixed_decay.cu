// fixed_decay.cu — linear recurrences with a matrix state per head and ONE constant decay per head (lightning attention, retention), over ragged
// batches with carried state:
//
//   S_t = a S_{t-1} + k_t v_t^T          o_t = S_t^T q_t
//
// The heads of a token are normed together afterwards.  That root mean square is one factor per token, so it need not be known before the
// out-projection: these kernels write o * weight * sigmoid(gate) and, per token and head, the square sum of o; the kernel that ends the sublayer divides the
// product by the root (residual.cu).  State fp32 [slots, heads, Dp, Vp]; a segment is (first row, rows, state slot, flags); positions[first row] == 0
// starts from zero whatever the slot holds.  q, k and v come with their activations.
//
//   k_fixed_chunk   many rows of bf16 models, chunks of 32 tokens on tensor cores
//   k_fixed_step    one row per segment
//   many rows in 32-bit: the sequential kernel of decay_scan.cu, then k_sums_gate
//
// k_fixed_chunk.  With S the state before a chunk of n tokens, numbered from 0:
//   o_t = a^(t+1) S^T q_t + sum_{s <= t} a^(t-s) (q_t . k_s) v_s          S <- a^n S + sum_s k_s (a^(n-1-s) v_s)^T
// Powers come from a table, so that nothing is divided.  S^T lies in the accumulators of the warps (16 value columns x all key channels each) and, as
// accumulator layout equals operand layout, is the left operand of the readout.  q, k and v are bf16 as they stand; fp32 operands are carried as sums of bf16
// numbers: a^(n-1-s) v_s as three (24 bits: the state is updated as in fp32), S and the 32 x 32 scores as two for results that end in bf16.
// Long segments are cut into groups that run in parallel: states of all groups but a segment's last from zero (STATE_ONLY), then the states they start
// from (k_fixed_starts), then all outputs.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>

#include "../pdl.cuh"
#include "attn_mma.cuh"
#include "decay.cuh"
#include "vec.cuh"

using namespace attn_mma;
using vec::from_f;
using vec::to_f;

namespace {

constexpr int kC = 32;

struct FixedParams {
  const void *q, *k, *v, *g;   // [rows, ld]: column h * Dp (q, k) or h * Vp (v, g) of each pointer
  const float* norm;           // [heads * Vp]
  const float* powers;         // [heads, kC + 1]: a^0 .. a^kC
  float* state;
  void* out;                   // [rows, ldo]
  float* sums;                 // [rows, nsum]
  const int *segs, *positions;
  int heads, Dp, Vp, ld, ldo, nsum;
};

template <int DK, int NW>
struct Shape {
  static constexpr int kPitch = DK * 2 + 16;                  // bytes; odd multiple of 16: ldmatrix without conflicts
  static constexpr int kVPitch = NW * 32 + 16;
  static constexpr int kAPitch = kC * 2 + 16;
  static constexpr int kOPitch = NW * 16 + 4;                 // floats
  static constexpr int oQ = 0;                                // [2 chunks][32][pitch]
  static constexpr int oK = oQ + 2 * kC * kPitch;
  static constexpr int oV = oK + 2 * kC * kPitch;
  static constexpr int oA = oV + 2 * kC * kVPitch;            // scores: hi, lo
  static constexpr int oO = oA + 2 * kC * kAPitch;            // o of a chunk, fp32
  static constexpr int oG = oO + kC * kOPitch * 4;            // gates of a chunk
  static constexpr int kBytes = oG + kC * kVPitch;
};

__device__ __forceinline__ float lo_f(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float hi_f(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }
// (x, y) = hi + lo, pairs of bf16; the rest is left in x and y
__device__ __forceinline__ uint32_t peel(float& x, float& y) {
  const uint32_t h = pack_bf16(x, y);
  x -= lo_f(h);
  y -= hi_f(h);
  return h;
}

template <int DK, int NW, bool STATE_ONLY>
__global__ void __launch_bounds__(NW * 32, DK > 128 ? 1 : 16 / NW) k_fixed_chunk(const FixedParams p, const int* groups, float* starts) {
  using S = Shape<DK, NW>;
  constexpr int NT = NW * 32;
  extern __shared__ __align__(16) uint8_t sm[];
  __shared__ float pw[kC + 1];
  pdl::launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r8 = lane >> 2, quad = lane & 3;
  const int h = blockIdx.y, gi = blockIdx.x;
  if (tid <= kC) pw[tid] = p.powers[h * (kC + 1) + tid];
  const uint32_t base = smem_addr(sm);
  // channels that the model does not have stay zeros
  for (int i = tid; i < 4 * kC * (DK - p.Dp) / 8; i += NT) {
    const int w = (DK - p.Dp) / 8, r = i / w;
    st_zero16(base + S::oQ + r * S::kPitch + (p.Dp + (i - r * w) * 8) * 2);
  }
  pdl::grid_dependency_wait();
  const int first = groups[4 * gi], n = groups[4 * gi + 1], slot = groups[4 * gi + 2], flags = groups[4 * gi + 3];
  if (STATE_ONLY && !(flags & 2)) return;
  const int vb = blockIdx.z * NW * 16, v0 = vb + warp * 16;         // first value column of the CTA, of the warp
  const bool mma_warp = v0 < p.Vp;
  const size_t hs = size_t(p.Dp) * p.Vp;                            // state values per head
  const __nv_bfloat16* qg = static_cast<const __nv_bfloat16*>(p.q) + size_t(h) * p.Dp;
  const __nv_bfloat16* kg = static_cast<const __nv_bfloat16*>(p.k) + size_t(h) * p.Dp;
  const __nv_bfloat16* vg = static_cast<const __nv_bfloat16*>(p.v) + size_t(h) * p.Vp + vb;
  const __nv_bfloat16* gg = static_cast<const __nv_bfloat16*>(p.g) + size_t(h) * p.Vp + vb;
  const int dch = p.Dp / 8, vch = min(NW * 16, p.Vp - vb) / 8;

  // rows of chunk c on their way to shared memory; missing rows are zeros
  auto issue = [&](int c) {
    const int at = c * kC, nt = min(kC, n - at);
    const uint32_t qb = base + S::oQ + (c & 1) * kC * S::kPitch, kb = base + S::oK + (c & 1) * kC * S::kPitch, vbuf = base + S::oV + (c & 1) * kC * S::kVPitch;
#pragma unroll
    for (int i = tid; i < kC * (DK / 8); i += NT) {
      const int t = i / (DK / 8), x = i % (DK / 8);
      const size_t src = size_t(first + at + t) * p.ld + x * 8;
      const uint32_t o = t * S::kPitch + x * 16;
      if (x >= dch) continue;
      if (t < nt) {
        if (!STATE_ONLY) cp_async16(qb + o, qg + src);
        cp_async16(kb + o, kg + src);
      } else {
        if (!STATE_ONLY) st_zero16(qb + o);
        st_zero16(kb + o);
      }
    }
#pragma unroll
    for (int i = tid; i < kC * NW * 2; i += NT) {
      const int t = i / (NW * 2), x = i % (NW * 2);
      if (x >= vch) continue;
      if (t < nt) cp_async16(vbuf + t * S::kVPitch + x * 16, vg + size_t(first + at + t) * p.ld + x * 8);
      else st_zero16(vbuf + t * S::kVPitch + x * 16);
    }
    cp_async_commit();
  };
  auto issue_gates = [&](int c) {
    const int at = c * kC, nt = min(kC, n - at);
#pragma unroll
    for (int i = tid; i < kC * NW * 2; i += NT) {
      const int t = i / (NW * 2), x = i % (NW * 2);
      if (x < vch && t < nt) cp_async16(base + S::oG + t * S::kVPitch + x * 16, gg + size_t(first + at + t) * p.ld + x * 8);
    }
    cp_async_commit();
  };
  // square sum, weight and gate of chunk c, whose o lies in shared memory; a row per NW lanes, 16 columns per lane
  auto emit = [&](int c) {
    const int t = tid / NW, v = tid % NW * 16;
    const bool row_ok = c * kC + t < n;
    const size_t row = size_t(first + c * kC + t);
    float ss = 0.f;
#pragma unroll
    for (int x = 0; x < 2; x++) {
      const int col = v + x * 8;
      if (row_ok && vb + col < p.Vp) {
        float f[8], g[8], w[8];
        vec::load8(reinterpret_cast<const float*>(sm + S::oO) + t * S::kOPitch + col, f);
        vec::load8(reinterpret_cast<const __nv_bfloat16*>(sm + S::oG + t * S::kVPitch) + col, g);
        vec::load8(p.norm + size_t(h) * p.Vp + vb + col, w);
#pragma unroll
        for (int e = 0; e < 8; e++) {
          ss = fmaf(f[e], f[e], ss);
          f[e] = f[e] * w[e] * vec::sigmoid<__nv_bfloat16>(g[e]);
        }
        vec::store8(static_cast<__nv_bfloat16*>(p.out) + row * p.ldo + size_t(h) * p.Vp + vb + col, f);
      }
    }
#pragma unroll
    for (int o = NW / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (tid % NW == 0 && row_ok) p.sums[row * p.nsum + h * gridDim.z + blockIdx.z] = ss;
  };

  issue(0);
  float st[DK / 8][4];      // S^T: value column v0 + r8 (+ 8), channels 8 i + 2 quad (+ 1)
  const bool fresh = p.positions[first] == 0;
  const float* from = flags ? starts + (size_t(gi) * p.heads + h) * hs : p.state + (size_t(slot) * p.heads + h) * hs;
  const bool zero = STATE_ONLY || !mma_warp || (!flags && fresh);
#pragma unroll
  for (int i = 0; i < DK / 8; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int d = i * 8 + quad * 2 + (j & 1), v = v0 + r8 + (j >> 1) * 8;
      st[i][j] = zero || d >= p.Dp ? 0.f : from[size_t(d) * p.Vp + v];
    }
  const uint32_t brow = (lane & 7) + ((lane >> 4) << 3), bcol = ((lane >> 3) & 1) * 16;    // right operands stored [n][k]
  const int nc = (n + kC - 1) / kC;
  for (int c = 0; c < nc; c++) {
    const int nt = min(kC, n - c * kC);
    const uint32_t qb = base + S::oQ + (c & 1) * kC * S::kPitch, kb = base + S::oK + (c & 1) * kC * S::kPitch, vbuf = base + S::oV + (c & 1) * kC * S::kVPitch;
    cp_async_wait<0>();
    __syncthreads();
    if (!STATE_ONLY && c > 0) emit(c - 1);
    if (c + 1 < nc) issue(c + 1);
    float o[kC / 8][4] = {};  // o^T: value column as above, tokens 8 i + 2 quad (+ 1)
    if (!STATE_ONLY) {
      // scores: six tiles of 16 x 8 at or below the diagonal
      for (int tile = warp; tile < 6; tile += NW) {
        const int m = tile < 2 ? 0 : 1, n8 = tile < 2 ? tile : tile - 2;
        float acc[2][4] = {};
#pragma unroll
        for (int ks = 0; ks < DK / 16; ks++) {
          uint32_t a[4], b[2];
          ldmatrix_x4(qb + (m * 16 + (lane & 15)) * S::kPitch + (lane >> 4) * 16 + ks * 32, a);
          ldmatrix_x2(kb + (n8 * 8 + (lane & 7)) * S::kPitch + ((lane >> 3) & 1) * 16 + ks * 32, b);
          mma_bf16(acc[ks & 1], a, b[0], b[1]);
        }
        const int s = n8 * 8 + quad * 2;
#pragma unroll
        for (int r = 0; r < 2; r++) {
          const int t = m * 16 + r8 + r * 8;
          float x = s <= t ? (acc[0][2 * r] + acc[1][2 * r]) * pw[max(t - s, 0)] : 0.f;
          float y = s + 1 <= t ? (acc[0][2 * r + 1] + acc[1][2 * r + 1]) * pw[max(t - s - 1, 0)] : 0.f;
          uint8_t* dst = sm + S::oA + t * S::kAPitch + s * 2;
          *reinterpret_cast<uint32_t*>(dst) = peel(x, y);
          *reinterpret_cast<uint32_t*>(dst + kC * S::kAPitch) = pack_bf16(x, y);
        }
      }
      if (mma_warp) {
#pragma unroll
        for (int ks = 0; ks < DK / 16; ks++) {
          uint32_t sh[4], sl[4];
#pragma unroll
          for (int r = 0; r < 4; r++) {
            float x = st[2 * ks + (r >> 1)][2 * (r & 1)], y = st[2 * ks + (r >> 1)][2 * (r & 1) + 1];
            sh[r] = peel(x, y);
            sl[r] = pack_bf16(x, y);
          }
          uint32_t b[kC / 16][4];
#pragma unroll
          for (int j = 0; j < kC / 16; j++) ldmatrix_x4(qb + (brow + 16 * j) * S::kPitch + bcol + ks * 32, b[j]);
#pragma unroll
          for (int j = 0; j < kC / 8; j++) mma_bf16(o[j], sl, b[j >> 1][2 * (j & 1)], b[j >> 1][2 * (j & 1) + 1]);
#pragma unroll
          for (int j = 0; j < kC / 8; j++) mma_bf16(o[j], sh, b[j >> 1][2 * (j & 1)], b[j >> 1][2 * (j & 1) + 1]);
        }
#pragma unroll
        for (int i = 0; i < kC / 8; i++) {
          const float e0 = pw[i * 8 + quad * 2 + 1], e1 = pw[i * 8 + quad * 2 + 2];
          o[i][0] *= e0; o[i][1] *= e1; o[i][2] *= e0; o[i][3] *= e1;
        }
      }
      __syncthreads();
      issue_gates(c);
    }
    if (mma_warp) {
      uint32_t vf[kC / 16][4];   // v^T: stored [token][column]
#pragma unroll
      for (int x = 0; x < kC / 16; x++)
        ldmatrix_x4_trans(vbuf + (x * 16 + brow) * S::kVPitch + (warp * 16 + ((lane >> 3) & 1) * 8) * 2, vf[x]);
      if (!STATE_ONLY) {
#pragma unroll
        for (int x = 0; x < kC / 16; x++)
#pragma unroll
          for (int j = x; j < kC / 16; j++)
#pragma unroll
            for (int part = 1; part >= 0; part--) {
              uint32_t b[4];
              ldmatrix_x4(base + S::oA + part * kC * S::kAPitch + (brow + 16 * j) * S::kAPitch + bcol + x * 32, b);
              mma_bf16(o[2 * j], vf[x], b[0], b[1]);
              mma_bf16(o[2 * j + 1], vf[x], b[2], b[3]);
            }
        float* so = reinterpret_cast<float*>(sm + S::oO) + warp * 16 + r8;
#pragma unroll
        for (int i = 0; i < kC / 8; i++)
#pragma unroll
          for (int j = 0; j < 4; j++) so[(i * 8 + quad * 2 + (j & 1)) * S::kOPitch + (j >> 1) * 8] = o[i][j];
      }
      const float e = pw[nt];
#pragma unroll
      for (int i = 0; i < DK / 8; i++) { st[i][0] *= e; st[i][1] *= e; st[i][2] *= e; st[i][3] *= e; }
#pragma unroll
      for (int x = 0; x < kC / 16; x++) {
        uint32_t w[3][4];         // a^(n-1-s) v_s^T in three parts
#pragma unroll
        for (int r = 0; r < 4; r++) {
          const int left = nt - 1 - (x * 16 + (r >> 1) * 8 + quad * 2);     // tokens after this one; rows past the end hold zeros
          float f0 = lo_f(vf[x][r]) * pw[max(left, 0)], f1 = hi_f(vf[x][r]) * pw[max(left - 1, 0)];
          w[0][r] = peel(f0, f1);
          w[1][r] = peel(f0, f1);
          w[2][r] = pack_bf16(f0, f1);
        }
#pragma unroll
        for (int i = 0; i < DK / 16; i += 2) {        // four accumulators in turn
          uint32_t b[2][4];
#pragma unroll
          for (int j = 0; j < 2; j++) ldmatrix_x4_trans(kb + (x * 16 + (lane & 15)) * S::kPitch + (i + j) * 32 + (lane >> 4) * 16, b[j]);
#pragma unroll
          for (int part = 2; part >= 0; part--)       // smallest part first
#pragma unroll
            for (int j = 0; j < 4; j++) mma_bf16(st[2 * i + j], w[part], b[j >> 1][2 * (j & 1)], b[j >> 1][2 * (j & 1) + 1]);
        }
      }
    }
  }
  if (!STATE_ONLY) {
    cp_async_wait<0>();
    __syncthreads();
    emit(nc - 1);
  }
  if (mma_warp && (STATE_ONLY || !(flags & 2))) {
    float* to = STATE_ONLY ? starts + (size_t(gi + 1) * p.heads + h) * hs : p.state + (size_t(slot) * p.heads + h) * hs;
#pragma unroll
    for (int i = 0; i < DK / 8; i++)
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const int d = i * 8 + quad * 2 + (j & 1), v = v0 + r8 + (j >> 1) * 8;
        if (d < p.Dp) to[size_t(d) * p.Vp + v] = st[i][j];
      }
  }
}

// Before: starts[g + 1] = the state that group g alone leaves (from zero).  After: starts[g] = the state that group g starts from.  One CTA column per
// segment of several groups (at its first group).
__global__ void __launch_bounds__(256) k_fixed_starts(const FixedParams p, const int* groups, float* starts) {
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  int g = blockIdx.x;
  const int h = blockIdx.y, i = blockIdx.z * 256 + threadIdx.x, hv = p.Dp * p.Vp / 4;
  if (groups[4 * g + 3] != 2 || i >= hv) return;
  const double a = double(p.powers[h * (kC + 1) + 1]);
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.positions[groups[4 * g]] != 0) s = reinterpret_cast<const float4*>(p.state)[(size_t(groups[4 * g + 2]) * p.heads + h) * hv + i];
  float4* at = reinterpret_cast<float4*>(starts) + (size_t(g) * p.heads + h) * hv + i;
  *at = s;
  int rows = -1;
  float e = 0.f;
  while (groups[4 * g + 3] & 2) {
    if (groups[4 * g + 1] != rows) {
      rows = groups[4 * g + 1];
      e = float(pow(a, double(rows)));
    }
    g++;
    at += size_t(p.heads) * hv;
    const float4 l = *at;
    s = make_float4(fmaf(e, s.x, l.x), fmaf(e, s.y, l.y), fmaf(e, s.z, l.z), fmaf(e, s.w, l.w));
    *at = s;
  }
}

// o fp32 [rows, heads * Vp] -> o * weight * sigmoid(gate) and square sums, one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) k_sums_gate(const FixedParams p, const float* o, int rows) {
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (w >= (long long)rows * p.heads) return;
  const int row = int(w / p.heads), h = int(w - (long long)row * p.heads);
  float ss = 0.f;
  for (int i = lane * 8; i < p.Vp; i += 256) {
    float f[8], g[8], wt[8];
    vec::load8(o + size_t(w) * p.Vp + i, f);
    vec::load8(static_cast<const T*>(p.g) + size_t(row) * p.ld + size_t(h) * p.Vp + i, g);
    vec::load8(p.norm + size_t(h) * p.Vp + i, wt);
#pragma unroll
    for (int e = 0; e < 8; e++) {
      ss = fmaf(f[e], f[e], ss);
      f[e] = f[e] * wt[e] * vec::sigmoid<T>(g[e]);
    }
    vec::store8(static_cast<T*>(p.out) + size_t(row) * p.ldo + size_t(h) * p.Vp + i, f);
  }
#pragma unroll
  for (int d = 16; d > 0; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
  if (lane == 0) p.sums[size_t(row) * p.nsum + h] = ss;
}

// One row per segment.  Threads: 4 value columns each, as many groups of keys as fit.
constexpr int kStepThreads = 256, kStepKeys = 16;
template <typename T>
__global__ void __launch_bounds__(kStepThreads) k_fixed_step(const FixedParams p) {
  extern __shared__ __align__(16) uint8_t sm[];
  __shared__ float red[8];
  const int h = blockIdx.x, tid = threadIdx.x, nc = p.Vp / 4, nkg = max(1, kStepThreads / nc);
  float *qs = reinterpret_cast<float*>(sm), *ks = qs + p.Dp, *acc = ks + p.Dp;
  pdl::launch_dependents();
  const float a = p.powers[h * (kC + 1) + 1];
  pdl::grid_dependency_wait();
  const int* seg = p.segs + 4 * blockIdx.y;
  const int row = seg[0], slot = seg[2];
  const bool fresh = p.positions[row] == 0;
  float4* st = reinterpret_cast<float4*>(p.state + (size_t(slot) * p.heads + h) * p.Dp * p.Vp);
  const int kgi = tid / nc, cg = tid - kgi * nc;
  const bool on = kgi < nkg;
  // the first keys of the state are requested before anything is computed
  float4 S[kStepKeys];
#pragma unroll
  for (int i = 0; i < kStepKeys; i++) {
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on && !fresh && kgi + i * nkg < p.Dp) S[i] = st[size_t(kgi + i * nkg) * nc + cg];
  }
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (on) {
    const T* vr = static_cast<const T*>(p.v) + size_t(row) * p.ld + size_t(h) * p.Vp + cg * 4;
    v = make_float4(to_f(vr[0]), to_f(vr[1]), to_f(vr[2]), to_f(vr[3]));
  }
  for (int d = tid; d < p.Dp; d += kStepThreads) {
    const size_t at = size_t(row) * p.ld + size_t(h) * p.Dp + d;
    qs[d] = to_f(static_cast<const T*>(p.q)[at]);
    ks[d] = to_f(static_cast<const T*>(p.k)[at]);
  }
  __syncthreads();
  if (on) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    auto one = [&](int key, float4 x) {
      const float q = qs[key], k = ks[key];
      x = make_float4(fmaf(a, x.x, k * v.x), fmaf(a, x.y, k * v.y), fmaf(a, x.z, k * v.z), fmaf(a, x.w, k * v.w));
      st[size_t(key) * nc + cg] = x;
      o.x = fmaf(q, x.x, o.x); o.y = fmaf(q, x.y, o.y); o.z = fmaf(q, x.z, o.z); o.w = fmaf(q, x.w, o.w);
    };
#pragma unroll
    for (int i = 0; i < kStepKeys; i++)
      if (kgi + i * nkg < p.Dp) one(kgi + i * nkg, S[i]);
#pragma unroll 8
    for (int key = kgi + kStepKeys * nkg; key < p.Dp; key += nkg) one(key, fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : st[size_t(key) * nc + cg]);
    *reinterpret_cast<float4*>(acc + kgi * p.Vp + cg * 4) = o;
  }
  __syncthreads();
  float sq = 0.f;
  for (int c = tid; c < p.Vp; c += kStepThreads) {
    float o = 0.f;
    for (int w = 0; w < nkg; w++) o += acc[w * p.Vp + c];
    sq = fmaf(o, o, sq);
    const size_t hv = size_t(h) * p.Vp + c;
    from_f(static_cast<T*>(p.out)[size_t(row) * p.ldo + hv], o * p.norm[hv] * vec::sigmoid<T>(to_f(static_cast<const T*>(p.g)[size_t(row) * p.ld + hv])));
  }
#pragma unroll
  for (int d = 16; d > 0; d >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, d);
  if ((tid & 31) == 0) red[tid >> 5] = sq;
  __syncthreads();
  if (tid == 0) {
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) tot += red[w];
    p.sums[size_t(row) * p.nsum + h] = tot;
  }
}

template <int DK, int NW, bool STATE_ONLY>
cudaError_t launch(const FixedParams& p, const int* groups, int ngroups, float* starts, cudaStream_t st) {
  static bool done = false;
  constexpr size_t smem = Shape<DK, NW>::kBytes;
  cudaError_t e = allow_smem(k_fixed_chunk<DK, NW, STATE_ONLY>, smem, &done);
  return e != cudaSuccess ? e : pdl::launch(k_fixed_chunk<DK, NW, STATE_ONLY>, dim3(ngroups, p.heads, (p.Vp / 16 + NW - 1) / NW), dim3(NW * 32), smem, st, 1, p, groups, starts);
}
template <int DK, int NW>
cudaError_t run(const FixedParams& p, const int* groups, int ngroups, bool multi, float* starts, cudaStream_t st) {
  cudaError_t e = cudaSuccess;
  if (multi) {
    e = launch<DK, NW, true>(p, groups, ngroups, starts, st);
    if (e == cudaSuccess) e = pdl::launch(k_fixed_starts, dim3(ngroups, p.heads, (p.Dp * p.Vp / 4 + 255) / 256), dim3(256), 0, st, 1, p, groups, starts);
  }
  return e != cudaSuccess ? e : launch<DK, NW, false>(p, groups, ngroups, starts, st);
}
template <int DK>
cudaError_t run(const FixedParams& p, const int* groups, int ngroups, bool multi, float* starts, cudaStream_t st) {
  return p.Vp <= 64 ? run<DK, 4>(p, groups, ngroups, multi, starts, st) : run<DK, 8>(p, groups, ngroups, multi, starts, st);
}
int value_blocks(int Vp) { return Vp <= 64 ? 1 : (Vp + 127) / 128; }

}  // namespace

extern "C" {

int tbv_op_fixed_decay_chunk(void) { return kC; }
// square sums per row that tbv_op_fixed_decay_scan writes
int tbv_op_fixed_decay_sums(int heads, int Vp, int bf16) { return bf16 ? heads * value_blocks(Vp) : heads; }

// Many rows.  powers [heads, chunk + 1] = a^0 .. a^chunk.  bf16: groups [ngroups, 4] are the segments, possibly cut (flags: 1 = a group of the same segment
// precedes, 2 = one follows); multi: some segment is cut, and starts [ngroups, heads, Dp, Vp] is scratch.  fp32: segs [nseg, 4], o = scratch [rows, heads * Vp].
int tbv_op_fixed_decay_scan(const void* q, const void* k, const void* v, const void* g, const void* norm, const void* powers, void* state, void* o, void* out,
                            void* sums, const void* segs, const void* positions, const void* groups, int ngroups, int multi, void* starts, int rows, int nseg, int heads,
                            int Dp, int Vp, int ld, int ldo, int bf16, void* stream) {
  if (rows <= 0 || nseg <= 0) return 0;
  if (!decay_ops::sizes_ok(heads, Dp, Vp) || nseg > 65535 || (ld % 8) || (ldo % 8) || (bf16 && (!groups || ngroups <= 0 || (multi && !starts))) || (!bf16 && !o)) return -2;
  FixedParams p{q, k, v, g, static_cast<const float*>(norm), static_cast<const float*>(powers), static_cast<float*>(state), out, static_cast<float*>(sums),
                static_cast<const int*>(segs), static_cast<const int*>(positions), heads, Dp, Vp, ld, ldo, tbv_op_fixed_decay_sums(heads, Vp, bf16)};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (bf16) {
    const int* gr = static_cast<const int*>(groups);
    float* s = static_cast<float*>(starts);
    if (Dp <= 32) e = run<32>(p, gr, ngroups, multi, s, st);
    else if (Dp <= 64) e = run<64>(p, gr, ngroups, multi, s, st);
    else if (Dp <= 128) e = run<128>(p, gr, ngroups, multi, s, st);
    else e = run<256>(p, gr, ngroups, multi, s, st);
  } else {
    decay_ops::ScanParams sp{};
    sp.q = q; sp.k = k; sp.v = v; sp.state = p.state; sp.o = static_cast<float*>(o); sp.segs = p.segs; sp.positions = p.positions;
    sp.heads = heads; sp.Dp = Dp; sp.Vp = Vp; sp.ld = ld; sp.qscale = 1.f; sp.fixed = p.powers + 1; sp.fixed_ld = kC + 1;
    e = decay_ops::sequential_scan_f32(sp, nseg, st);
    if (e == cudaSuccess) e = pdl::launch(k_sums_gate<float>, dim3(unsigned(((long long)rows * heads + 7) / 8)), dim3(256), 0, st, 1, p, static_cast<const float*>(o), rows);
  }
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] fixed-decay scan launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

// One row per segment; sums [rows, heads].
int tbv_op_fixed_decay_step(const void* q, const void* k, const void* v, const void* g, const void* norm, const void* powers, void* state, void* out, void* sums,
                            const void* segs, const void* positions, int nseg, int heads, int Dp, int Vp, int ld, int ldo, int bf16, void* stream) {
  if (nseg <= 0) return 0;
  if (!decay_ops::sizes_ok(heads, Dp, Vp) || nseg > 65535) return -2;
  FixedParams p{q, k, v, g, static_cast<const float*>(norm), static_cast<const float*>(powers), static_cast<float*>(state), out, static_cast<float*>(sums),
                static_cast<const int*>(segs), static_cast<const int*>(positions), heads, Dp, Vp, ld, ldo, heads};
  const int nc = Vp / 4, nkg = nc < kStepThreads ? kStepThreads / nc : 1;
  const size_t smem = size_t(2 * Dp + nkg * Vp) * 4;        // at most 10 KB
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = bf16 ? pdl::launch(k_fixed_step<__nv_bfloat16>, dim3(heads, nseg), dim3(kStepThreads), smem, st, 1, p)
                       : pdl::launch(k_fixed_step<float>, dim3(heads, nseg), dim3(kStepThreads), smem, st, 1, p);
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] fixed-decay step launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

}  // extern "C"
