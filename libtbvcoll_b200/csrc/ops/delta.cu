// delta.cu — gated delta rule with a decay per key channel, over ragged batches with carried state.  Per head, with q and k made unit vectors (q also scaled by
// 1 / sqrt(dim)):
//
//   S' = diag(a_t) S_{t-1}      u_t = beta_t (v_t - S'^T k_t)      S_t = S' + k_t u_t^T      o_t = S_t^T q_t = S'^T q_t + (q_t . k_t) u_t
//   a = exp(-rate * softplus(z)),  beta = sigmoid(.),  out = o / rms(o) * weight * sigmoid(gate)
//
// so that one pass over the decayed state gives both readouts.  A segment (first row, rows, state slot) may be a whole prompt, a portion or one token;
// positions[first row] == 0 starts from zero whatever the slot holds.  State fp32 [slots, heads, Dp, Vp]; all of this is fp32 arithmetic.
//
//   delta_chunk.cu  many rows of bf16 models, on tensor cores; k_delta_scan is its 32-bit counterpart
//   k_delta_scan    many rows, token by token: a CTA walks one segment for one head and a block of value columns, S in registers (packed pairs of keys)
//   k_delta_step    one row per segment: a CTA per (head, row) with the convolution, the low-rank products of decays and gates, and norm and gate behind the step
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>

#include "../pdl.cuh"
#include "attn_mma.cuh"
#include "delta.cuh"
#include "ops.h"

using namespace vec;
using delta_ops::decay;
using delta_ops::kUnitEps;
using delta_ops::Params;

namespace {

constexpr int kChunk = 16, kVT = 4;

template <typename T, int KG, int KT>
__global__ void __launch_bounds__(128) k_delta_scan(const Params p) {
  constexpr int DK = KG * KT, COLS = 4 * (32 / KG) * kVT, NP = KT / 2;
  extern __shared__ __align__(16) float sm[];
  float *qs = sm, *ks = qs + kChunk * DK, *as = ks + kChunk * DK, *vs = as + kChunk * DK, *os = vs + kChunk * COLS, *bt = os + kChunk * COLS, *qk = bt + kChunk;
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kg = lane % KG;
  const int h = blockIdx.y, g = h / (p.heads / p.kv_heads), c0 = blockIdx.x * COLS, cl = (warp * (32 / KG) + lane / KG) * kVT;
  const int* seg = p.segs + 4 * blockIdx.z;
  const int first = seg[0], n = seg[1], slot = seg[2];
  const bool fresh = p.positions[first] == 0;
  const float rate = p.rate[h], qscale = rsqrtf(float(p.dim));
  float* st = p.state + (size_t(slot) * p.heads + h) * p.Dp * p.Vp + c0;

  // S: pairs of keys 4 * (kg + KG * j) + 2 * (i & 1) .., pair i = 2 * j + (i & 1)
  f32x2 S[NP][kVT];
#pragma unroll
  for (int i = 0; i < NP; i++) {
    const int key = 4 * (kg + KG * (i >> 1)) + 2 * (i & 1);
#pragma unroll
    for (int c = 0; c < kVT; c++) {
      const bool in = !fresh && key < p.Dp && c0 + cl + c < p.Vp;
      S[i][c] = in ? pack2(st[size_t(key) * p.Vp + cl + c], st[size_t(key + 1) * p.Vp + cl + c]) : 0ull;
    }
  }
  for (int at = 0; at < n; at += kChunk) {
    const int nt = min(kChunk, n - at);
    __syncthreads();
    for (int t = warp; t < nt; t += 4) {
      const size_t r = size_t(first + at + t);
      const T *q = static_cast<const T*>(p.q) + r * p.ld + size_t(g) * p.Dp, *k = static_cast<const T*>(p.k) + r * p.ld + size_t(g) * p.Dp;
      const float* z = p.z + r * p.ldz + size_t(h) * p.Dp;
      float sq = 0.f, sk = 0.f, s = 0.f;
      for (int d = lane; d < DK; d += 32) {
        const bool in = d < p.Dp;
        const float qv = in ? to_f(q[d]) : 0.f, kv = in ? to_f(k[d]) : 0.f;
        qs[t * DK + d] = qv;
        ks[t * DK + d] = kv;
        as[t * DK + d] = in ? decay<T>(z[d], rate) : 1.f;
        sq = fmaf(qv, qv, sq);
        sk = fmaf(kv, kv, sk);
        s = fmaf(qv, kv, s);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
        s += __shfl_xor_sync(0xffffffffu, s, o);
      }
      const float fq = qscale / sqrtf(sq + kUnitEps), fk = 1.f / sqrtf(sk + kUnitEps);
      for (int d = lane; d < DK; d += 32) { qs[t * DK + d] *= fq; ks[t * DK + d] *= fk; }
      if (lane == 0) {
        bt[t] = sigmoid<T>(to_f(static_cast<const T*>(p.beta)[r * p.ldx + h]));
        qk[t] = s * fq * fk;
      }
      const T* v = static_cast<const T*>(p.v) + r * p.ld + size_t(h) * p.Vp + c0;
      for (int c = lane; c < COLS; c += 32) vs[t * COLS + c] = c0 + c < p.Vp ? to_f(v[c]) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < nt; t++) {
      f32x2 k2[NP], ak[kVT], aq[kVT];
#pragma unroll
      for (int c = 0; c < kVT; c++) ak[c] = aq[c] = 0ull;
#pragma unroll
      for (int j = 0; j < KT / 4; j++) {
        const int x = t * DK + 4 * (kg + KG * j);
        const ulonglong2 va = *reinterpret_cast<const ulonglong2*>(as + x), vk = *reinterpret_cast<const ulonglong2*>(ks + x), vq = *reinterpret_cast<const ulonglong2*>(qs + x);
        k2[2 * j] = vk.x;
        k2[2 * j + 1] = vk.y;
#pragma unroll
        for (int c = 0; c < kVT; c++) {
          S[2 * j][c] = mul2(va.x, S[2 * j][c]);
          S[2 * j + 1][c] = mul2(va.y, S[2 * j + 1][c]);
          ak[c] = fma2(vk.y, S[2 * j + 1][c], fma2(vk.x, S[2 * j][c], ak[c]));
          aq[c] = fma2(vq.y, S[2 * j + 1][c], fma2(vq.x, S[2 * j][c], aq[c]));
        }
      }
      float sk[kVT], sq[kVT];
#pragma unroll
      for (int c = 0; c < kVT; c++) {
        float lo, hi;
        unpack2(ak[c], lo, hi);
        sk[c] = lo + hi;
        unpack2(aq[c], lo, hi);
        sq[c] = lo + hi;
#pragma unroll
        for (int o = KG / 2; o > 0; o >>= 1) {
          sk[c] += __shfl_xor_sync(0xffffffffu, sk[c], o);
          sq[c] += __shfl_xor_sync(0xffffffffu, sq[c], o);
        }
        const float u = bt[t] * (vs[t * COLS + cl + c] - sk[c]);
        const f32x2 uu = pack2(u, u);
#pragma unroll
        for (int i = 0; i < NP; i++) S[i][c] = fma2(k2[i], uu, S[i][c]);
        if (kg == c) os[t * COLS + cl + c] = fmaf(qk[t], u, sq[c]);
      }
    }
    __syncthreads();
    for (int i = tid; i < nt * (COLS / 4); i += 128) {
      const int t = i / (COLS / 4), c = i % (COLS / 4) * 4;
      if (c0 + c < p.Vp)
        *reinterpret_cast<float4*>(p.o + size_t(first + at + t) * p.heads * p.Vp + size_t(h) * p.Vp + c0 + c) = *reinterpret_cast<const float4*>(os + t * COLS + c);
    }
  }
#pragma unroll
  for (int i = 0; i < NP; i++) {
    const int key = 4 * (kg + KG * (i >> 1)) + 2 * (i & 1);
#pragma unroll
    for (int c = 0; c < kVT; c++)
      if (key < p.Dp && c0 + cl + c < p.Vp) {
        float lo, hi;
        unpack2(S[i][c], lo, hi);
        st[size_t(key) * p.Vp + cl + c] = lo;
        st[size_t(key + 1) * p.Vp + cl + c] = hi;
      }
  }
}

// out = o / rms(o) * weight * sigmoid(gate), one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) k_delta_norm_gate(const Params p, int rows) {
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (w >= (long long)rows * p.heads) return;
  const int row = int(w / p.heads), h = int(w - (long long)row * p.heads);
  const float* o = p.o + size_t(w) * p.Vp;
  float ss = 0.f;
  for (int i = lane * 8; i < p.Vp; i += 256) {
    float f[8];
    load8(o + i, f);
#pragma unroll
    for (int e = 0; e < 8; e++) ss = fmaf(f[e], f[e], ss);      // pad columns hold zeros
  }
#pragma unroll
  for (int d = 16; d > 0; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
  const float r = 1.0f / sqrtf(ss / float(p.vdim) + p.eps);
  for (int i = lane * 8; i < p.Vp; i += 256) {
    float f[8], g[8], wt[8];
    load8(o + i, f);
    load8(static_cast<const T*>(p.gate) + size_t(row) * p.ldg + size_t(h) * p.Vp + i, g);
    load8(p.norm + i, wt);
#pragma unroll
    for (int e = 0; e < 8; e++) f[e] = f[e] * r * wt[e] * sigmoid<T>(g[e]);
    store8(static_cast<T*>(p.out) + size_t(row) * p.ldo + size_t(h) * p.Vp + i, f);
  }
}

// One row per segment.  Threads: 4 value columns each, as many groups of keys as fit.
constexpr int kStepThreads = 256, kStepKeys = 16, kStepTaps = 3;     // kStepTaps: carried inputs of the convolution taken at once
template <typename T>
__global__ void __launch_bounds__(kStepThreads) k_delta_step(const Params p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[4][8];
  const int h = blockIdx.x, g = h / (p.heads / p.kv_heads), tid = threadIdx.x, nc = p.Vp / 4, nkg = max(1, kStepThreads / nc);
  float *qs = sm, *ks = qs + p.Dp, *vs = ks + p.Dp, *as = vs + p.Vp, *us = as + p.Dp, *gs = us + p.Vp, *acc = gs + p.Vp, *la = acc + 2 * nkg * p.Vp, *lg = la + p.rank;
  pdl::launch_dependents();
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
  for (int i = tid; i < 2 * p.rank; i += kStepThreads)
    la[i] = to_f((i < p.rank ? static_cast<const T*>(p.low_a) : static_cast<const T*>(p.low_g) - p.rank)[size_t(row) * p.ldx + i]);
  // q, k, v of this head; the convolution over the carried inputs first, if it was not done before
  float sq = 0.f, sk = 0.f, sd = 0.f;
  // (all loads of a thread's two values come before its stores: one round trip)
  const int K = p.kv_heads * p.Dp, total = 2 * p.Dp + p.Vp, keep = p.taps_w ? p.taps - 1 : 0;
  for (int i0 = tid; i0 < total; i0 += 2 * kStepThreads) {
    float cur[2], in[2][kStepTaps], w[2][kStepTaps], last[2];
    int column[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int i = i0 + e * kStepThreads;
      if (i >= total) continue;
      const int part = i < p.Dp ? 0 : (i < 2 * p.Dp ? 1 : 2), c = part == 2 ? h * p.Vp + i - 2 * p.Dp : g * p.Dp + i - part * p.Dp;
      column[e] = part * K + c;
      cur[e] = to_f((part == 0 ? static_cast<const T*>(p.q) : (part == 1 ? static_cast<const T*>(p.k) : static_cast<const T*>(p.v)))[size_t(row) * p.ld + c]);
      if (!p.taps_w) continue;
      last[e] = p.taps_w[size_t(keep) * p.C + column[e]];
      const float* past = p.conv + size_t(slot) * keep * p.C + column[e];
#pragma unroll
      for (int j = 0; j < kStepTaps; j++) {
        in[e][j] = j < keep && !fresh ? past[size_t(j) * p.C] : 0.f;
        w[e][j] = j < keep ? p.taps_w[size_t(j) * p.C + column[e]] : 0.f;
      }
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int i = i0 + e * kStepThreads;
      if (i >= total) continue;
      float v = cur[e];
      if (p.taps_w) {
        float* past = p.conv + size_t(slot) * keep * p.C + column[e];
        float a = 0.f;
#pragma unroll
        for (int j = 0; j < kStepTaps; j++) {
          a = fmaf(w[e][j], in[e][j], a);
          if (j > 0 && j < keep) past[size_t(j - 1) * p.C] = in[e][j];
        }
        for (int j = kStepTaps; j < keep; j++) {
          const float x = fresh ? 0.f : past[size_t(j) * p.C];
          a = fmaf(p.taps_w[size_t(j) * p.C + column[e]], x, a);
          past[size_t(j - 1) * p.C] = x;
        }
        a = fmaf(last[e], v, a);
        if (keep) past[size_t(keep - 1) * p.C] = v;
        T o;
        from_f(o, vec::gate<T>(a));              // rounded as where the convolution is a kernel of its own
        v = to_f(o);
      }
      qs[i] = v;                                 // q, k and v one after the other
    }
  }
  __syncthreads();
  const float rate = p.rate[h];
  for (int i = tid; i < p.Dp + p.Vp; i += kStepThreads) {
    const bool dec = i < p.Dp;
    const int at = dec ? i : i - p.Dp;
    const size_t hd = dec ? size_t(h) * p.Dp + at : size_t(h) * p.Vp + at;
    const T* w2 = static_cast<const T*>(dec ? p.w_a : p.w_g) + hd * p.rank;
    const float* low = dec ? la : lg;
    float s = dec ? to_f(static_cast<const T*>(p.b_a)[hd]) : 0.f;
#pragma unroll 4
    for (int r = 0; r < p.rank; r += 8) {
      float w[8];
      load8(w2 + r, w);
#pragma unroll
      for (int e = 0; e < 8; e++) s = fmaf(low[r + e], w[e], s);
    }
    if (dec) as[at] = decay<T>(softplus<T>(s), rate);
    else gs[at] = sigmoid<T>(s);
  }
  for (int d = tid; d < p.Dp; d += kStepThreads) {
    sq = fmaf(qs[d], qs[d], sq);
    sk = fmaf(ks[d], ks[d], sk);
    sd = fmaf(qs[d], ks[d], sd);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sk += __shfl_xor_sync(0xffffffffu, sk, o);
    sd += __shfl_xor_sync(0xffffffffu, sd, o);
  }
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; red[2][tid >> 5] = sd; }
  __syncthreads();
  sq = sk = sd = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) { sq += red[0][w]; sk += red[1][w]; sd += red[2][w]; }
  const float fq = rsqrtf(float(p.dim)) / sqrtf(sq + kUnitEps), fk = 1.f / sqrtf(sk + kUnitEps);
  if (on) {
    float4 ok = make_float4(0.f, 0.f, 0.f, 0.f), oq = ok;
    auto read = [&](int key, float4& x) {
      const float a = as[key], q = qs[key], k = ks[key];
      x = make_float4(a * x.x, a * x.y, a * x.z, a * x.w);
      ok.x = fmaf(k, x.x, ok.x); ok.y = fmaf(k, x.y, ok.y); ok.z = fmaf(k, x.z, ok.z); ok.w = fmaf(k, x.w, ok.w);
      oq.x = fmaf(q, x.x, oq.x); oq.y = fmaf(q, x.y, oq.y); oq.z = fmaf(q, x.z, oq.z); oq.w = fmaf(q, x.w, oq.w);
    };
#pragma unroll
    for (int i = 0; i < kStepKeys; i++)
      if (kgi + i * nkg < p.Dp) read(kgi + i * nkg, S[i]);
    if (!fresh)
      for (int key = kgi + kStepKeys * nkg; key < p.Dp; key += nkg) {
        float4 x = st[size_t(key) * nc + cg];
        read(key, x);
      }
    *reinterpret_cast<float4*>(acc + kgi * p.Vp + cg * 4) = ok;
    *reinterpret_cast<float4*>(acc + (nkg + kgi) * p.Vp + cg * 4) = oq;
  }
  __syncthreads();
  const float beta = sigmoid<T>(to_f(static_cast<const T*>(p.beta)[size_t(row) * p.ldx + h]));
  float ov[4], so = 0.f;                     // columns tid, tid + 256, .. (Vp <= 1024)
#pragma unroll
  for (int j = 0; j < 4; j++) {
    const int c = tid + j * kStepThreads;
    ov[j] = 0.f;
    if (c < p.Vp) {
      float ok = 0.f, oq = 0.f;
      for (int w = 0; w < nkg; w++) { ok += acc[w * p.Vp + c]; oq += acc[(nkg + w) * p.Vp + c]; }
      const float u = beta * (vs[c] - fk * ok);
      us[c] = fk * u;
      ov[j] = fmaf(fq * fk * sd, u, fq * oq);
      so = fmaf(ov[j], ov[j], so);
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) so += __shfl_xor_sync(0xffffffffu, so, o);
  if ((tid & 31) == 0) red[3][tid >> 5] = so;
  __syncthreads();
  if (on) {
    const float4 u = *reinterpret_cast<const float4*>(us + cg * 4);
    auto write = [&](int key, const float4& x) {
      const float k = ks[key];
      st[size_t(key) * nc + cg] = make_float4(fmaf(k, u.x, x.x), fmaf(k, u.y, x.y), fmaf(k, u.z, x.z), fmaf(k, u.w, x.w));
    };
#pragma unroll
    for (int i = 0; i < kStepKeys; i++)
      if (kgi + i * nkg < p.Dp) write(kgi + i * nkg, S[i]);
    for (int key = kgi + kStepKeys * nkg; key < p.Dp; key += nkg) {
      const float a = as[key];
      const float4 x = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : st[size_t(key) * nc + cg];
      write(key, make_float4(a * x.x, a * x.y, a * x.z, a * x.w));
    }
  }
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) tot += red[3][w];
  const float r = 1.0f / sqrtf(tot / float(p.vdim) + p.eps);
#pragma unroll
  for (int j = 0; j < 4; j++) {
    const int c = tid + j * kStepThreads;
    if (c < p.Vp) from_f(static_cast<T*>(p.out)[size_t(row) * p.ldo + size_t(h) * p.Vp + c], ov[j] * r * p.norm[c] * gs[c]);
  }
}

template <typename T, int KG, int KT>
cudaError_t launch_scan(const Params& p, int nseg, cudaStream_t st) {
  constexpr int COLS = 4 * (32 / KG) * kVT;
  constexpr size_t smem = size_t(kChunk * (3 * KG * KT + 2 * COLS + 2)) * 4;
  static bool done = false;
  cudaError_t e = attn_mma::allow_smem(k_delta_scan<T, KG, KT>, smem, &done);
  return e != cudaSuccess ? e : pdl::launch(k_delta_scan<T, KG, KT>, dim3((p.Vp + COLS - 1) / COLS, p.heads, nseg), dim3(128), smem, st, 1, p);
}
template <typename T>
cudaError_t scan(const Params& p, int nseg, cudaStream_t st) {
  if (p.Dp <= 32) return launch_scan<T, 8, 4>(p, nseg, st);
  if (p.Dp <= 64) return launch_scan<T, 8, 8>(p, nseg, st);
  if (p.Dp <= 128) return launch_scan<T, 16, 8>(p, nseg, st);
  return launch_scan<T, 32, 8>(p, nseg, st);
}

}  // namespace

extern "C" {

// Many rows per segment: q, k, v [rows, ld] behind convolution and SiLU, beta [rows, ldb], z fp32 [rows, ldz] = softplus of the decay inputs, gate [rows, ldg]; o fp32 scratch [rows, heads * Vp].
// groups (bf16; null: the sequential kernel): the segments as the chunked kernels take them, [ngroups, 4]; sets: scratch of tbv_op_delta_sets bytes, or null (see
// delta_chunk.cu).
int tbv_op_delta_scan(const void* q, const void* k, const void* v, const void* beta, const void* z, const void* gate, const void* rate, const void* norm,
                      void* state, void* o, void* out, const void* segs, const void* positions, const void* groups, int ngroups, void* sets, int rows, int nseg, int heads,
                      int kv_heads, int Dp, int Vp, int dim, int vdim, int ld, int ldb, int ldz, int ldg, int ldo, float eps, int bf16, void* stream) {
  if (rows <= 0 || nseg <= 0) return 0;
  Params p{};
  p.q = q; p.k = k; p.v = v; p.beta = beta; p.z = static_cast<const float*>(z); p.gate = gate; p.rate = static_cast<const float*>(rate);
  p.norm = static_cast<const float*>(norm); p.state = static_cast<float*>(state); p.o = static_cast<float*>(o); p.out = out;
  p.segs = static_cast<const int*>(segs); p.positions = static_cast<const int*>(positions);
  p.heads = heads; p.kv_heads = kv_heads; p.Dp = Dp; p.Vp = Vp; p.dim = dim; p.vdim = vdim; p.ld = ld; p.ldx = ldb; p.ldz = ldz; p.ldg = ldg; p.ldo = ldo; p.eps = eps;
  if (!delta_ops::sizes_ok(p) || nseg > 65535 || (ld % 8) || (ldz % 8) || (ldg % 8) || (ldo % 8)) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  bool finished = false;
  if (bf16 && groups && delta_ops::chunk_fits(p)) e = delta_ops::chunk_scan(p, static_cast<const int*>(groups), ngroups, rows, sets, &finished, st);
  else e = bf16 ? scan<__nv_bfloat16>(p, nseg, st) : scan<float>(p, nseg, st);
  if (e == cudaSuccess && !finished) {
    const dim3 grid(unsigned(((long long)rows * heads + 7) / 8));
    e = bf16 ? pdl::launch(k_delta_norm_gate<__nv_bfloat16>, grid, dim3(256), 0, st, 1, p, rows) : pdl::launch(k_delta_norm_gate<float>, grid, dim3(256), 0, st, 1, p, rows);
  }
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] delta scan launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

// Bytes of `sets` that the form for few sequences and heads needs; 0: the sizes do not take the chunked kernels, or the GPU is busy enough without it.
long long tbv_op_delta_sets(int rows, int ngroups, int heads, int Dp, int Vp) {
  Params p{};
  p.heads = heads; p.Dp = Dp; p.Vp = Vp;
  if (!delta_ops::chunk_fits(p) || 2 * ngroups * heads * ((Vp + 127) / 128) > tbvops::sm_count()) return 0;
  return (long long)delta_ops::chunk_sets(p, rows, ngroups);
}

// One row per segment.  beta, low_a, low_g: columns of rows ldx apart; w_a [heads * Dp, rank], b_a [heads * Dp], w_g [heads * Vp, rank].  taps_w [taps, C] (C = the
// q, k and v columns) and conv [slots, taps - 1, C]: q, k, v are taken before the convolution and the carried inputs are replaced (every key head has one
// query head then); null: q, k, v are behind it.
int tbv_op_delta_step(const void* q, const void* k, const void* v, const void* beta, const void* low_a, const void* low_g, const void* w_a, const void* b_a,
                      const void* w_g, const void* rate, const void* norm, void* state, void* out, const void* taps_w, void* conv, const void* segs,
                      const void* positions, int nseg, int heads, int kv_heads, int Dp, int Vp, int dim, int vdim, int ld, int ldx, int rank, int taps, int ldo, float eps,
                      int bf16, void* stream) {
  if (nseg <= 0) return 0;
  Params p{};
  p.q = q; p.k = k; p.v = v; p.beta = beta; p.low_a = low_a; p.low_g = low_g; p.w_a = w_a; p.b_a = b_a; p.w_g = w_g; p.rate = static_cast<const float*>(rate);
  p.norm = static_cast<const float*>(norm); p.state = static_cast<float*>(state); p.out = out; p.taps_w = static_cast<const float*>(taps_w); p.conv = static_cast<float*>(conv);
  p.segs = static_cast<const int*>(segs); p.positions = static_cast<const int*>(positions);
  p.heads = heads; p.kv_heads = kv_heads; p.Dp = Dp; p.Vp = Vp; p.dim = dim; p.vdim = vdim; p.ld = ld; p.ldx = ldx; p.rank = rank; p.taps = taps; p.ldo = ldo; p.eps = eps;
  p.C = 2 * kv_heads * Dp + heads * Vp;
  if (!delta_ops::sizes_ok(p) || nseg > 65535 || rank <= 0 || (rank % 8) || rank > 1024 || (taps_w && (taps < 1 || heads != kv_heads || (taps > 1 && !conv)))) return -2;
  const int nc = Vp / 4, nkg = nc < kStepThreads ? kStepThreads / nc : 1;
  const size_t smem = size_t(3 * Dp + 3 * Vp + 2 * nkg * Vp + 2 * rank) * 4;        // at most 32 KB
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = bf16 ? pdl::launch(k_delta_step<__nv_bfloat16>, dim3(heads, nseg), dim3(kStepThreads), smem, st, 1, p)
                       : pdl::launch(k_delta_step<float>, dim3(heads, nseg), dim3(kStepThreads), smem, st, 1, p);
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] delta step launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

}  // extern "C"
