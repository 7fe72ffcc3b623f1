// decay_scan.cu — linear recurrences with a matrix state per head and a decay per key channel, over ragged batches with carried state:
//
//   o_t = S_{t-1}^T q'_t + s_t v_t          S_t = diag(a_t) S_{t-1} + k_t v_t^T
//
//   gated linear attention   q' = a * q, s = q . k   (the state is read after the update)     a = sigmoid(z)^(1 / tau)
//   WKV                      q' = r,     s = r . (u * k)   (before it, the bonus u aside)     a = exp(-exp(z))
//
// and per head  out = o / rms(o) * weight * silu(gate).  A segment (first row, rows, state slot) may be a whole prompt, a portion or one
// token; positions[first row] == 0 starts from zero whatever the slot holds.  State fp32 [slots, heads, Dp, Vp]; all of it is fp32 arithmetic.
//
//   chunk_scan.cu  many rows of bf16 models, on tensor cores; k_decay_scan is its 32-bit counterpart
//   k_decay_scan   many rows: a CTA walks one segment for one head and a block of value columns.  A thread keeps KT keys x VT columns of S
//                  in registers (packed pairs of keys); rows come in chunks whose decays are made once per chunk in shared memory.  The sums
//                  over keys cross KG lanes by halving.  o goes to memory in fp32 and k_head_norm_gate finishes it.
//   k_decay_step   one row per segment: a CTA per (head, row) with the low-rank decay product before and norm and gate behind the step.
// The last kernel of the layer to read the previous token's input replaces it (shift): the recurrence is that kernel.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>

#include "../pdl.cuh"
#include "attn_mma.cuh"
#include "decay.cuh"
#include "ops.h"
#include "vec.cuh"

using namespace vec;
using decay_ops::decay;
using decay_ops::ScanParams;

namespace {

template <int DK, int COLS>
struct ScanShape {
  static constexpr int C = DK > 128 ? 8 : 16;       // rows per chunk
  static constexpr int U8 = DK / 8, V8 = COLS / 8;
  static constexpr int NU = (C * U8 + 127) / 128, NV = (C * V8 + 127) / 128;
  static constexpr int kFloats = C * (3 * DK + 2 * COLS + U8 + 1) + C;
};

template <typename T, int KG, int KT, int VT>
__global__ void __launch_bounds__(128) k_decay_scan(const ScanParams p) {
  constexpr int DK = KG * KT, COLS = 4 * (32 / KG) * VT;
  using Sh = ScanShape<DK, COLS>;
  constexpr int C = Sh::C, U8 = Sh::U8, V8 = Sh::V8, NU = Sh::NU, NV = Sh::NV, NP = KT / 2;
  extern __shared__ __align__(16) float sm[];
  float *qs = sm, *ks = qs + C * DK, *as = ks + C * DK, *vs = as + C * DK, *os = vs + C * COLS, *part = os + C * COLS, *ss = part + C * (U8 + 1);
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kg = lane % KG;
  const int h = blockIdx.y, c0 = blockIdx.x * COLS, cl = (warp * (32 / KG) + lane / KG) * VT;   // first column of this thread in the CTA
  const int* seg = p.segs + 4 * blockIdx.z;
  const int first = seg[0], n = seg[1], slot = seg[2];
  const bool fresh = p.positions[first] == 0, wkv = p.u != nullptr;
  const float fixed = p.fixed ? p.fixed[h * p.fixed_ld] : 0.f;
  const T* qp = static_cast<const T*>(p.q) + size_t(h) * p.Dp;
  const T* kp = static_cast<const T*>(p.k) + size_t(h) * p.Dp;
  const T* vp = static_cast<const T*>(p.v) + size_t(h) * p.Vp + c0;
  float* st = p.state + (size_t(slot) * p.heads + h) * p.Dp * p.Vp + c0;

  Raw8<T> rq[NU], rk[NU], rv[NV];
  Raw8<float> rz[NU];
  auto issue = [&](int at) {
#pragma unroll
    for (int i = 0; i < NU; i++) {
      const int u = tid + i * 128, t = u / U8, d = u % U8 * 8;
      if (u < C * U8 && at + t < n && d < p.Dp) {
        const size_t r = size_t(first + at + t);
        rq[i].load(qp + r * p.ld + d);
        rk[i].load(kp + r * p.ld + d);
        if (!p.fixed) rz[i].load(p.z + r * p.ldz + size_t(h) * p.Dp + d);
      }
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int u = tid + i * 128, t = u / V8, c = u % V8 * 8;
      if (u < C * V8 && at + t < n && c0 + c < p.Vp) rv[i].load(vp + size_t(first + at + t) * p.ld + c);
    }
  };
  issue(0);

  // S: pairs of keys 4 * (kg + KG * j) + 2 * (i & 1) .., pair i = 2 * j + (i & 1)
  f32x2 S[NP][VT];
#pragma unroll
  for (int i = 0; i < NP; i++) {
    const int key = 4 * (kg + KG * (i >> 1)) + 2 * (i & 1);
#pragma unroll
    for (int c = 0; c < VT; c++) {
      const bool in = !fresh && key < p.Dp && c0 + cl + c < p.Vp;
      S[i][c] = in ? pack2(st[size_t(key) * p.Vp + cl + c], st[size_t(key + 1) * p.Vp + cl + c]) : 0ull;
    }
  }

  for (int at = 0; at < n; at += C) {
    const int nt = min(C, n - at);
#pragma unroll
    for (int i = 0; i < NU; i++) {
      const int u = tid + i * 128, t = u / U8, d = u % U8 * 8;
      if (u < C * U8 && t < nt) {
        float q[8] = {}, k[8] = {}, a[8], s = 0.f;
        if (d < p.Dp) {
          float z[8];
          rq[i].unpack(q);
          rk[i].unpack(k);
          if (!p.fixed) rz[i].unpack(z);
#pragma unroll
          for (int e = 0; e < 8; e++) {
            a[e] = p.fixed ? fixed : decay<T>(z[e], wkv, p.inv_tau);
            if (wkv) {
              s = fmaf(q[e] * p.u[h * p.Dp + d + e], k[e], s);
            } else {
              q[e] *= p.qscale;
              s = fmaf(q[e], k[e], s);
              q[e] *= a[e];
            }
          }
        } else {
#pragma unroll
          for (int e = 0; e < 8; e++) a[e] = 1.f;
        }
        store8(qs + t * DK + d, q);
        store8(ks + t * DK + d, k);
        store8(as + t * DK + d, a);
        part[t * (U8 + 1) + d / 8] = s;
      }
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int u = tid + i * 128, t = u / V8, c = u % V8 * 8;
      if (u < C * V8 && t < nt) {
        float v[8] = {};
        if (c0 + c < p.Vp) rv[i].unpack(v);
        store8(vs + t * COLS + c, v);
      }
    }
    __syncthreads();
    if (tid < nt) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < U8; i++) s += part[tid * (U8 + 1) + i];
      ss[tid] = s;
    }
    issue(at + C);
    __syncthreads();
#pragma unroll 2
    for (int t = 0; t < nt; t++) {
      f32x2 a2[NP], k2[NP], q2[NP];
#pragma unroll
      for (int j = 0; j < KT / 4; j++) {
        const int x = t * DK + 4 * (kg + KG * j);
        const ulonglong2 va = *reinterpret_cast<const ulonglong2*>(as + x), vk = *reinterpret_cast<const ulonglong2*>(ks + x), vq = *reinterpret_cast<const ulonglong2*>(qs + x);
        a2[2 * j] = va.x; a2[2 * j + 1] = va.y;
        k2[2 * j] = vk.x; k2[2 * j + 1] = vk.y;
        q2[2 * j] = vq.x; q2[2 * j + 1] = vq.y;
      }
      float v[VT], o[VT];
#pragma unroll
      for (int c = 0; c < VT; c += 4) {
        const float4 f = *reinterpret_cast<const float4*>(vs + t * COLS + cl + c);
        v[c] = f.x; v[c + 1] = f.y; v[c + 2] = f.z; v[c + 3] = f.w;
      }
#pragma unroll
      for (int c = 0; c < VT; c++) {
        const f32x2 vv = pack2(v[c], v[c]);
        f32x2 acc = mul2(q2[0], S[0][c]);
        S[0][c] = fma2(a2[0], S[0][c], mul2(k2[0], vv));
#pragma unroll
        for (int i = 1; i < NP; i++) {
          acc = fma2(q2[i], S[i][c], acc);
          S[i][c] = fma2(a2[i], S[i][c], mul2(k2[i], vv));
        }
        float lo, hi;
        unpack2(acc, lo, hi);
        o[c] = lo + hi;
      }
      // sums over the KG lanes: halve the columns while there are several, then plain exchanges
      int col = 0;
#pragma unroll
      for (int w = VT, off = KG / 2; off >= 1; off >>= 1) {
        if (w > 1) {
          const bool up = lane & off;
#pragma unroll
          for (int j = 0; j < VT / 2; j++)
            if (j < w / 2) {
              const float send = up ? o[j] : o[j + w / 2], keep = up ? o[j + w / 2] : o[j];
              o[j] = keep + __shfl_xor_sync(0xffffffffu, send, off);
            }
          w >>= 1;
          if (up) col += w;
        } else {
          o[0] += __shfl_xor_sync(0xffffffffu, o[0], off);
        }
      }
      if ((lane & (KG / VT - 1)) == 0) os[t * COLS + cl + col] = fmaf(ss[t], vs[t * COLS + cl + col], o[0]);
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
    for (int c = 0; c < VT; c++)
      if (key < p.Dp && c0 + cl + c < p.Vp) {
        float lo, hi;
        unpack2(S[i][c], lo, hi);
        st[size_t(key) * p.Vp + cl + c] = lo;
        st[size_t(key + 1) * p.Vp + cl + c] = hi;
      }
  }
  if (p.h1) {
    const int ctas = gridDim.x * gridDim.y, id = blockIdx.y * gridDim.x + blockIdx.x;
    for (int i = id * 128 + tid; i < p.ldh; i += ctas * 128) p.shift[size_t(slot) * p.ldh + i] = p.h1[size_t(first + n - 1) * p.ldh + i];
  }
}

// out = o / rms(o) * weight * silu(gate), one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) k_head_norm_gate(const ScanParams p, int rows) {
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
    load8(static_cast<const T*>(p.g) + size_t(row) * p.ld + size_t(h) * p.Vp + i, g);
    load8(p.norm + size_t(h) * p.Vp + i, wt);
#pragma unroll
    for (int e = 0; e < 8; e++) f[e] = f[e] * r * wt[e] * gate<T>(g[e]);
    store8(static_cast<T*>(p.out) + size_t(row) * p.ldo + size_t(h) * p.Vp + i, f);
  }
}

// One row per segment.  Threads: 4 value columns each, as many groups of keys as fit.
constexpr int kStepThreads = 256, kStepKeys = 16;
template <typename T>
__global__ void __launch_bounds__(kStepThreads) k_decay_step(const ScanParams p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[8];
  const int h = blockIdx.x, tid = threadIdx.x, nc = p.Vp / 4, nkg = max(1, kStepThreads / nc);
  float *qs = sm, *ks = qs + p.Dp, *as = ks + p.Dp, *vs = as + p.Dp, *acc = vs + p.Vp, *low = acc + nkg * p.Vp;
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int* seg = p.segs + 4 * blockIdx.y;
  const int row = seg[0], slot = seg[2];
  const bool fresh = p.positions[row] == 0, wkv = p.u != nullptr;
  float4* st = reinterpret_cast<float4*>(p.state + (size_t(slot) * p.heads + h) * p.Dp * p.Vp);
  const int kgi = tid / nc, cg = tid - kgi * nc;
  const bool on = kgi < nkg;
  // the first keys of the state are requested before anything is computed
  float4 S[kStepKeys];
  if (on && !fresh) {
#pragma unroll
    for (int i = 0; i < kStepKeys; i++)
      if (kgi + i * nkg < p.Dp) S[i] = st[size_t(kgi + i * nkg) * nc + cg];
  } else {
#pragma unroll
    for (int i = 0; i < kStepKeys; i++) S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int i = tid; i < p.rank; i += kStepThreads) {
    const float f = to_f(static_cast<const T*>(p.low)[size_t(row) * p.ldlow + i]);
    low[i] = wkv ? tanhf(f) : f;
  }
  for (int i = tid; i < p.Vp; i += kStepThreads) vs[i] = to_f(static_cast<const T*>(p.v)[size_t(row) * p.ld + size_t(h) * p.Vp + i]);
  __syncthreads();
  float s = 0.f;
  for (int d = tid; d < p.Dp; d += kStepThreads) {
    const size_t hd = size_t(h) * p.Dp + d;
    float z = to_f(static_cast<const T*>(p.b2)[hd]);
    for (int r = 0; r < p.rank; r += 8) {
      float w[8];
      load8(static_cast<const T*>(p.w2) + hd * p.rank + r, w);
#pragma unroll
      for (int e = 0; e < 8; e++) z = fmaf(low[r + e], w[e], z);
    }
    const float a = decay<T>(z, wkv, p.inv_tau);
    float q = to_f(static_cast<const T*>(p.q)[size_t(row) * p.ld + hd]);
    const float k = to_f(static_cast<const T*>(p.k)[size_t(row) * p.ld + hd]);
    if (wkv) {
      s = fmaf(q * p.u[hd], k, s);
    } else {
      q *= p.qscale;
      s = fmaf(q, k, s);
      q *= a;
    }
    qs[d] = q;
    ks[d] = k;
    as[d] = a;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  if ((tid & 31) == 0) red[tid >> 5] = s;
  __syncthreads();
  float sum = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) sum += red[w];
  if (on) {
    const float4 v = *reinterpret_cast<const float4*>(vs + cg * 4);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    auto one = [&](int key, float4 x) {
      const float q = qs[key], k = ks[key], a = as[key];
      o.x = fmaf(q, x.x, o.x); o.y = fmaf(q, x.y, o.y); o.z = fmaf(q, x.z, o.z); o.w = fmaf(q, x.w, o.w);
      st[size_t(key) * nc + cg] = make_float4(fmaf(a, x.x, k * v.x), fmaf(a, x.y, k * v.y), fmaf(a, x.z, k * v.z), fmaf(a, x.w, k * v.w));
    };
#pragma unroll
    for (int i = 0; i < kStepKeys; i++)
      if (kgi + i * nkg < p.Dp) one(kgi + i * nkg, S[i]);
#pragma unroll 8
    for (int key = kgi + kStepKeys * nkg; key < p.Dp; key += nkg) one(key, fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : st[size_t(key) * nc + cg]);
    *reinterpret_cast<float4*>(acc + kgi * p.Vp + cg * 4) = o;
  }
  __syncthreads();
  float ov[4], sq = 0.f;                     // columns tid, tid + 256, .. (Vp <= 1024)
#pragma unroll
  for (int j = 0; j < 4; j++) {
    const int c = tid + j * kStepThreads;
    ov[j] = 0.f;
    if (c < p.Vp) {
      float o = 0.f;
      for (int w = 0; w < nkg; w++) o += acc[w * p.Vp + c];
      ov[j] = fmaf(sum, vs[c], o);
      sq = fmaf(ov[j], ov[j], sq);
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
  if ((tid & 31) == 0) red[tid >> 5] = sq;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) tot += red[w];
  const float r = 1.0f / sqrtf(tot / float(p.vdim) + p.eps);
#pragma unroll
  for (int j = 0; j < 4; j++) {
    const int c = tid + j * kStepThreads;
    if (c < p.Vp) {
      const float g = to_f(static_cast<const T*>(p.g)[size_t(row) * p.ld + size_t(h) * p.Vp + c]);
      from_f(static_cast<T*>(p.out)[size_t(row) * p.ldo + size_t(h) * p.Vp + c], ov[j] * r * p.norm[size_t(h) * p.Vp + c] * gate<T>(g));
    }
  }
}

template <typename T, int KG, int KT, int VT>
cudaError_t launch_scan(const ScanParams& p, int nseg, cudaStream_t st) {
  constexpr int COLS = 4 * (32 / KG) * VT;
  constexpr size_t smem = size_t(ScanShape<KG * KT, COLS>::kFloats) * 4;
  static bool done = false;
  cudaError_t e = attn_mma::allow_smem(k_decay_scan<T, KG, KT, VT>, smem, &done);
  return e != cudaSuccess ? e : pdl::launch(k_decay_scan<T, KG, KT, VT>, dim3((p.Vp + COLS - 1) / COLS, p.heads, nseg), dim3(128), smem, st, 1, p);
}
template <typename T, int KG, int KT>
cudaError_t scan_columns(const ScanParams& p, int nseg, cudaStream_t st) {
  // eight columns per thread need two warps per scheduler to hide latencies; with fewer segments four columns make twice as many
  constexpr int COLS = 4 * (32 / KG) * 8;
  const long warps = 4l * nseg * p.heads * ((p.Vp + COLS - 1) / COLS);
  if (p.Vp <= COLS / 2 || warps < 8l * tbvops::sm_count()) return launch_scan<T, KG, KT, 4>(p, nseg, st);
  return launch_scan<T, KG, KT, 8>(p, nseg, st);
}
template <typename T>
cudaError_t scan(const ScanParams& p, int nseg, cudaStream_t st) {
  if (p.Dp <= 32) return scan_columns<T, 8, 4>(p, nseg, st);
  if (p.Dp <= 64) return scan_columns<T, 8, 8>(p, nseg, st);
  if (p.Dp <= 128) return scan_columns<T, 16, 8>(p, nseg, st);
  return scan_columns<T, 32, 8>(p, nseg, st);
}
bool sizes_ok(int heads, int Dp, int Vp, int vdim) { return decay_ops::sizes_ok(heads, Dp, Vp) && vdim <= Vp; }

}  // namespace

namespace decay_ops {
cudaError_t sequential_scan_f32(const ScanParams& p, int nseg, cudaStream_t st) { return scan<float>(p, nseg, st); }
}  // namespace decay_ops

extern "C" {

// Many rows per segment: recurrence (o fp32 scratch [rows, heads * Vp]), then head norm and gate.  u != null: WKV.  h1 / shift: see the top.
// groups (bf16; null: the sequential kernel): the segments cut for the chunked kernels (chunk_scan.cu), [ngroups, 4]; `multi` tells whether any segment
// has several; starts [ngroups, heads, Dp, Vp] and totals [ngroups, heads, Dp] fp32 are their scratch.  With groups, z may be null: then
// z = low . w2 + b2 inside (low [rows, ldlow] as it enters the product, w2 [heads * Dp, rank], rank a multiple of 16 and at most 128).
int tbv_op_decay_scan(const void* q, const void* k, const void* v, const void* g, const void* z, const void* u, const void* norm, void* state,
                      void* o, void* out, const void* h1, void* shift, const void* segs, const void* positions, const void* groups, int ngroups, int multi,
                      void* starts, void* totals, const void* low, const void* w2, const void* b2, int ldlow, int rank, int rows, int nseg, int heads, int Dp,
                      int Vp, int vdim, int ld, int ldz, int ldo, int ldh, float qscale, float tau, float eps, int bf16, void* stream) {
  if (rows <= 0 || nseg <= 0) return 0;
  if (!sizes_ok(heads, Dp, Vp, vdim) || nseg > 65535 || (ld % 8) || (ldz % 8) || (ldo % 8) || !(tau > 0.f)) return -2;
  if (!z && (!bf16 || !groups || rank <= 0 || (rank % 16) || rank > decay_ops::kMaxRank || (ldlow % 8))) return -2;
  ScanParams p{};
  p.q = q; p.k = k; p.v = v; p.g = g; p.z = static_cast<const float*>(z); p.u = static_cast<const float*>(u); p.norm = static_cast<const float*>(norm);
  p.state = static_cast<float*>(state); p.o = static_cast<float*>(o); p.out = out; p.h1 = static_cast<const float*>(h1); p.shift = static_cast<float*>(shift);
  p.segs = static_cast<const int*>(segs); p.positions = static_cast<const int*>(positions);
  p.heads = heads; p.Dp = Dp; p.Vp = Vp; p.vdim = vdim; p.ld = ld; p.ldz = ldz; p.ldo = ldo; p.ldh = ldh;
  p.low = low; p.w2 = w2; p.b2 = b2; p.ldlow = ldlow; p.rank = rank;
  p.qscale = qscale; p.inv_tau = 1.0f / tau; p.eps = eps;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  bool finished = false;
  if (bf16 && groups) e = decay_ops::chunk_scan(p, static_cast<const int*>(groups), ngroups, multi, static_cast<float*>(starts), static_cast<float*>(totals), &finished, st);
  else e = bf16 ? scan<__nv_bfloat16>(p, nseg, st) : scan<float>(p, nseg, st);
  if (e == cudaSuccess && !finished) {
    const dim3 grid(unsigned(((long long)rows * heads + 7) / 8));
    e = bf16 ? pdl::launch(k_head_norm_gate<__nv_bfloat16>, grid, dim3(256), 0, st, 1, p, rows) : pdl::launch(k_head_norm_gate<float>, grid, dim3(256), 0, st, 1, p, rows);
  }
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] decay scan launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

// One row per segment, with the second decay product: z = act(low) . w2 + b2 (act = tanh for WKV), w2 [heads * Dp, rank].
int tbv_op_decay_step(const void* q, const void* k, const void* v, const void* g, const void* low, const void* w2, const void* b2, const void* u,
                      const void* norm, void* state, void* out, const void* segs, const void* positions, int nseg, int heads, int Dp, int Vp, int vdim,
                      int ld, int ldlow, int rank, int ldo, float qscale, float tau, float eps, int bf16, void* stream) {
  if (nseg <= 0) return 0;
  if (!sizes_ok(heads, Dp, Vp, vdim) || nseg > 65535 || rank <= 0 || (rank % 8) || rank > 1024 || (ld % 8) || !(tau > 0.f)) return -2;
  ScanParams p{};
  p.q = q; p.k = k; p.v = v; p.g = g; p.low = low; p.w2 = w2; p.b2 = b2; p.u = static_cast<const float*>(u); p.norm = static_cast<const float*>(norm);
  p.state = static_cast<float*>(state); p.out = out; p.segs = static_cast<const int*>(segs); p.positions = static_cast<const int*>(positions);
  p.heads = heads; p.Dp = Dp; p.Vp = Vp; p.vdim = vdim; p.ld = ld; p.ldlow = ldlow; p.rank = rank; p.ldo = ldo;
  p.qscale = qscale; p.inv_tau = 1.0f / tau; p.eps = eps;
  const int nc = Vp / 4, nkg = nc < kStepThreads ? kStepThreads / nc : 1;
  const size_t smem = size_t(3 * Dp + Vp + nkg * Vp + rank) * 4;        // at most 16 KB
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = bf16 ? pdl::launch(k_decay_step<__nv_bfloat16>, dim3(heads, nseg), dim3(kStepThreads), smem, st, 1, p)
                       : pdl::launch(k_decay_step<float>, dim3(heads, nseg), dim3(kStepThreads), smem, st, 1, p);
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] decay step launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

}  // extern "C"
