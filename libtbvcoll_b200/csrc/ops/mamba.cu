// mamba.cu — short causal convolution and selective scan over ragged batches with carried state.
//
// A batch holds the rows of several sequences, each sequence's rows consecutive: a segment (first row, row count, state
// slot).  A segment may be a whole prompt, a portion of one or a single decoded token; positions[first row] == 0 marks the
// start of a sequence, whose state is zero whatever the slot holds.  Per slot and layer run the state is
//   conv  fp32 [taps - 1][ldc]   the convolution's last inputs, oldest first
//   ssm   fp32 [inner][N]        S of the recurrence
// Every kernel reads the state that earlier launches left; k_selective_scan, the last to run for a layer, replaces both.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../pdl.cuh"
#include "vec.cuh"

namespace {

using namespace vec;

struct ConvParams {
  const void* x;             // [rows, ldx], the first `ldc` columns are the convolution's inputs
  void* out;                 // [rows, ldo]
  const float* taps_w;       // [taps, ldc], row taps - 1 weighs the current token
  const float* bias;         // [ldc]
  const float* conv_state;   // [slots, taps - 1, ldc]
  const int* segs;           // [nseg, 4]
  const int* seg_of_row;     // [rows] or null (row i = segment i)
  const int* positions;      // [rows]
  int rows, ldx, ldo, ldc, taps;
};

// out = silu(bias + sum_k w[k] * input at distance taps - 1 - k).  A thread owns R consecutive rows of 8 channels.  Rows whose inputs
// all lie in their own segment share a sliding window of loads (TAPS > 0); the others look at each input on its own.
template <typename T, int TAPS, int R>
__global__ void __launch_bounds__(128) k_causal_conv_silu(const ConvParams p) {
  pdl::launch_dependents();
  const int c8 = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  const int taps = TAPS > 0 ? TAPS : p.taps;
  float bias[8], w[TAPS > 0 ? TAPS : 1][8];
  if (c8 < p.ldc) {                         // weights: no need to wait for the kernel before
    load8(p.bias + c8, bias);
#pragma unroll
    for (int k = 0; k < TAPS; k++) load8(p.taps_w + size_t(k) * p.ldc + c8, w[k]);
  }
  pdl::grid_dependency_wait();
  if (c8 >= p.ldc) return;
  const T* x = static_cast<const T*>(p.x);
  const int t0 = blockIdx.y * R;
  if (R > 1 && TAPS > 0 && t0 >= TAPS - 1 && t0 + R <= p.rows) {
    // the window is requested before it is known whether the rows share a segment
    Raw8<T> win[TAPS > 0 ? TAPS + R - 1 : 1];
#pragma unroll
    for (int i = 0; i < TAPS + R - 1; i++) win[i].load(x + size_t(t0 - (TAPS - 1) + i) * p.ldx + c8);
    const int sa = p.seg_of_row ? p.seg_of_row[t0] : t0, sb = p.seg_of_row ? p.seg_of_row[t0 + R - 1] : t0 + R - 1;
    if (sa == sb && t0 - p.segs[4 * sa] >= taps - 1) {
#pragma unroll
      for (int r = 0; r < R; r++) {
        float acc[8], v[8];
#pragma unroll
        for (int i = 0; i < 8; i++) acc[i] = bias[i];
#pragma unroll
        for (int k = 0; k < TAPS; k++) {
          win[r + k].unpack(v);
#pragma unroll
          for (int i = 0; i < 8; i++) acc[i] = fmaf(w[k][i], v[i], acc[i]);
        }
#pragma unroll
        for (int i = 0; i < 8; i++) acc[i] = gate<T>(acc[i]);
        store8(static_cast<T*>(p.out) + size_t(t0 + r) * p.ldo + c8, acc);
      }
      return;
    }
  }
  for (int r = 0; r < R; r++) {
    const int t = t0 + r;
    if (t >= p.rows) return;
    const int* sg = p.segs + 4 * (p.seg_of_row ? p.seg_of_row[t] : t);
    const int first = sg[0], slot = sg[2], j = t - first;
    const bool fresh = p.positions[first] == 0;
    const float* cs = p.conv_state + size_t(slot) * (taps - 1) * p.ldc + c8;
    float acc[8];
#pragma unroll
    for (int i = 0; i < 8; i++) acc[i] = bias[i];
#pragma unroll
    for (int k = 0; k < (TAPS > 0 ? TAPS : taps); k++) {
      const int back = taps - 1 - k;
      float v[8], wk[8];
      if (back <= j) load8(x + size_t(t - back) * p.ldx + c8, v);
      else load8(cs + size_t(taps - 1 + j - back) * p.ldc, v);
      if (TAPS == 0) load8(p.taps_w + size_t(k) * p.ldc + c8, wk);
      const bool none = back > j && fresh;       // before the sequence: zero, whatever the slot holds
#pragma unroll
      for (int i = 0; i < 8; i++) acc[i] = fmaf(TAPS > 0 ? w[TAPS > 0 ? k : 0][i] : wk[i], none ? 0.f : v[i], acc[i]);
    }
#pragma unroll
    for (int i = 0; i < 8; i++) acc[i] = gate<T>(acc[i]);
    store8(static_cast<T*>(p.out) + size_t(t) * p.ldo + c8, acc);
  }
}

struct ScanParams {
  const void* u;          // [rows, ldu]   convolved input
  const void* xz;         // [rows, ldxz]  convolution input (columns 0..) and gate (columns zoff ..)
  const float* dt;        // [rows, lddt]  step sizes before the softplus
  const float* bc;        // [rows, ldbc]  B at column boff, C at column coff
  const float* a2;        // [inner, N]    -exp(A_log) * log2(e)
  const float* d;         // [inner]
  float* ssm;             // [slots, inner, N]
  float* conv_state;      // [slots, taps - 1, ldc]
  void* out;              // [rows, ldo]   y * silu(gate)
  const int* segs;        // [nseg, 4]
  const int* positions;
  int inner, N, ldu, ldxz, zoff, lddt, ldbc, boff, coff, ldo, ldc, taps;
};

// Replaces the convolution state of channel c by its last taps - 1 inputs; ascending, so an old entry is read before it is overwritten.
template <typename T>
__device__ __forceinline__ void roll_conv_state(const ScanParams& p, const T* xz, int first, int count, int slot, bool fresh, int c) {
  float* cs = p.conv_state + size_t(slot) * (p.taps - 1) * p.ldc + c;
  for (int k = 0; k < p.taps - 1; k++) {
    const int j = count - (p.taps - 1) + k;
    cs[size_t(k) * p.ldc] = j >= 0 ? to_f(xz[(size_t(first) + j) * p.ldxz + c]) : (fresh ? 0.f : cs[size_t(k + count) * p.ldc]);
  }
}

// LPC lanes share a channel, NPL states each (LPC * NPL >= N); a CTA owns 128 / LPC channels of one segment and walks its
// rows in tiles of TT: the tile's inputs are staged in shared memory while the next tile's are already on their way
// in registers.  Inside a tile TB steps form a block: their decays are computed together (they do not depend on the state),
// the recurrence runs over them, and the TB partial sums over the states are added across the LPC lanes by a transposing
// butterfly that leaves every lane with the sums of its own steps.
template <typename T, int LPC, int NPL>
__global__ void __launch_bounds__(128) k_selective_scan(const ScanParams p) {
  constexpr int kC = 128 / LPC, NP = LPC * NPL;
  constexpr int TB = LPC <= 4 ? 4 : (LPC >= 16 ? 16 : LPC);
  constexpr int TT = LPC == 1 ? 8 : (LPC == 2 || NP >= 256 ? 16 : 32);
  constexpr int TS = TT + 4, YS = kC + 32 / LPC;
  constexpr int EX = (TT * kC + 127) / 128, EB = (TT * NP + 127) / 128;
  __shared__ __align__(16) float sdt[kC][TS], sdx[kC][TS];
  __shared__ float su[TT][kC], sg[TT][kC], sy[TT][YS], sd[kC];
  __shared__ __align__(16) float sb[TT][NP];
  __shared__ __align__(16) float sc[TT][NP];
  pdl::launch_dependents();
  const int c0 = blockIdx.x * kC, cl = threadIdx.x / LPC, c = c0 + cl, lane = threadIdx.x % LPC, n0 = lane * NPL;
  const bool active = c < p.inner;
  constexpr int NQ = NPL / 2;
  f32x2 a[NQ], s[NQ];
#pragma unroll
  for (int i = 0; i < NQ; i++) {
    const float* ap = p.a2 + size_t(c) * p.N + n0 + 2 * i;
    a[i] = pack2(active && n0 + 2 * i < p.N ? ap[0] : 0.f, active && n0 + 2 * i + 1 < p.N ? ap[1] : 0.f);
  }
  if (threadIdx.x < kC) sd[threadIdx.x] = c0 + int(threadIdx.x) < p.inner ? p.d[c0 + threadIdx.x] : 0.f;
  pdl::grid_dependency_wait();
  const int* seg = p.segs + 4 * blockIdx.y;
  const int first = seg[0], count = seg[1], slot = seg[2];
  const bool fresh = p.positions[first] == 0;
  const T* u = static_cast<const T*>(p.u);
  const T* xz = static_cast<const T*>(p.xz);
  float* sp = p.ssm + (size_t(slot) * p.inner + c) * p.N + n0;
#pragma unroll
  for (int i = 0; i < NQ; i++)
    s[i] = pack2(active && n0 + 2 * i < p.N && !fresh ? sp[2 * i] : 0.f, active && n0 + 2 * i + 1 < p.N && !fresh ? sp[2 * i + 1] : 0.f);

  // raw values: nothing here depends on a load before the next tile is staged
  T ru[EX], rg[EX], zero;
  from_f(zero, 0.f);
  float rd[EX], rb[EB], rc[EB];
  // element e of this thread: row tx + e * kRX of the tile, channel c0 + cx (and row tn + .., state nn + .. of B and C)
  constexpr int kRX = 128 / kC;
  const int tx = threadIdx.x / kC, cx = threadIdx.x % kC;
  const bool cok = c0 + cx < p.inner;
  const T* pu = u + (size_t(first) + tx) * p.ldu + c0 + cx;
  const T* pz = xz + (size_t(first) + tx) * p.ldxz + p.zoff + c0 + cx;
  const float* pd = p.dt + (size_t(first) + tx) * p.lddt + c0 + cx;
  const float* pb = p.bc + size_t(first) * p.ldbc;
  auto fetch = [&](int t0) {
#pragma unroll
    for (int e = 0; e < EX; e++) {
      const int t = tx + e * kRX;
      const bool ok = cok && t < TT && t0 + t < count;
      ru[e] = ok ? pu[e * kRX * p.ldu] : zero;
      rd[e] = ok ? pd[e * kRX * p.lddt] : 0.f;
      rg[e] = ok ? pz[e * kRX * p.ldxz] : zero;
    }
#pragma unroll
    for (int e = 0; e < EB; e++) {
      const int id = threadIdx.x + e * 128, t = id / NP, n = id % NP;
      const bool ok = id < TT * NP && t0 + t < count && n < p.N;
      rb[e] = ok ? pb[t * p.ldbc + p.boff + n] : 0.f;
      rc[e] = ok ? pb[t * p.ldbc + p.coff + n] : 0.f;
    }
    pu += size_t(TT) * p.ldu;
    pz += size_t(TT) * p.ldxz;
    pd += size_t(TT) * p.lddt;
    pb += size_t(TT) * p.ldbc;
  };
  T* po = static_cast<T*>(p.out) + (size_t(first) + tx) * p.ldo + c0 + cx;
  fetch(0);
  for (int t0 = 0; t0 < count; t0 += TT) {
    const int nt = min(TT, count - t0);
    __syncthreads();
#pragma unroll
    for (int e = 0; e < EX; e++) {
      const int t = tx + e * kRX, cc = cx;
      if (t < TT) {
        // rows past the end get a zero step: they leave the state as it is
        const float dt = t < nt ? softplus<T>(rd[e]) : 0.f;
        sdt[cc][t] = dt;
        const float uv = to_f(ru[e]);
        sdx[cc][t] = dt * uv;
        su[t][cc] = uv;
        sg[t][cc] = gate<T>(to_f(rg[e]));
      }
    }
#pragma unroll
    for (int e = 0; e < EB; e++) {
      const int id = threadIdx.x + e * 128;
      if (id < TT * NP) {
        sb[id / NP][id % NP] = rb[e];
        sc[id / NP][id % NP] = rc[e];
      }
    }
    __syncthreads();
    if (t0 + TT < count) fetch(t0 + TT);
    for (int tb = 0; tb < nt; tb += TB) {
      float y[TB];
#pragma unroll
      for (int q = 0; q < TB; q += 4) {
        const float4 dt4 = *reinterpret_cast<const float4*>(&sdt[cl][tb + q]), dx4 = *reinterpret_cast<const float4*>(&sdx[cl][tb + q]);
        const float dts[4] = {dt4.x, dt4.y, dt4.z, dt4.w}, dxs[4] = {dx4.x, dx4.y, dx4.z, dx4.w};
#pragma unroll
        for (int j = 0; j < 4; j++) {
          f32x2 bv[NQ], cv[NQ];
          if constexpr (NQ == 1) {
            bv[0] = *reinterpret_cast<const f32x2*>(&sb[tb + q + j][n0]);
            cv[0] = *reinterpret_cast<const f32x2*>(&sc[tb + q + j][n0]);
          } else {
#pragma unroll
            for (int i = 0; i < NQ; i += 2) {
              const ulonglong2 b4 = *reinterpret_cast<const ulonglong2*>(&sb[tb + q + j][n0 + 2 * i]), c4 = *reinterpret_cast<const ulonglong2*>(&sc[tb + q + j][n0 + 2 * i]);
              bv[i] = b4.x; bv[i + 1] = b4.y;
              cv[i] = c4.x; cv[i + 1] = c4.y;
            }
          }
          const f32x2 dt2 = pack2(dts[j], dts[j]), dx2 = pack2(dxs[j], dxs[j]);
          f32x2 acc2 = 0ull;
#pragma unroll
          for (int i = 0; i < NQ; i++) {
            float e0, e1;
            unpack2(mul2(dt2, a[i]), e0, e1);
            s[i] = fma2(pack2(pow2<T>(e0), pow2<T>(e1)), s[i], mul2(dx2, bv[i]));
            acc2 = i == 0 ? mul2(s[0], cv[0]) : fma2(s[i], cv[i], acc2);
          }
          float acc, acc_hi;
          unpack2(acc2, acc, acc_hi);
          acc += acc_hi;
          y[q + j] = acc;
        }
      }
      // transposing butterfly: at each level a lane keeps the half of the steps its bit selects and sends the other
      int n = TB, base = 0;
#pragma unroll
      for (int o = LPC / 2; o > 0; o >>= 1) {
        const bool up = (lane & o) != 0;
        if (n > 1) {
          n >>= 1;
#pragma unroll
          for (int j = 0; j < TB / 2; j++) {
            if (j < n) {
              const float give = up ? y[j] : y[j + n], keep = up ? y[j + n] : y[j];
              y[j] = keep + __shfl_xor_sync(0xffffffffu, give, o);
            }
          }
          base += up ? n : 0;
        } else {
          y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
        }
      }
#pragma unroll
      for (int j = 0; j < TB; j++)
        if (j < n) sy[tb + base + j][cl] = y[j];
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < EX; e++) {
      const int t = tx + e * kRX;
      if (t < nt && cok) from_f(po[e * kRX * p.ldo], fmaf(sd[cx], su[t][cx], sy[t][cx]) * sg[t][cx]);
    }
    po += size_t(TT) * p.ldo;
  }
#pragma unroll
  for (int i = 0; i < NQ; i++) {
    float lo, hi;
    unpack2(s[i], lo, hi);
    if (active && n0 + 2 * i < p.N) sp[2 * i] = lo;
    if (active && n0 + 2 * i + 1 < p.N) sp[2 * i + 1] = hi;
  }
  if (active && lane == 0) roll_conv_state(p, xz, first, count, slot, fresh, c);
}

// One token per segment (a decode step): everything a thread needs is requested at once.
template <typename T, int LPC, int NPL>
__global__ void __launch_bounds__(128) k_scan_step(const ScanParams p) {
  pdl::launch_dependents();
  const int c = blockIdx.x * (128 / LPC) + threadIdx.x / LPC, lane = threadIdx.x % LPC, n0 = lane * NPL;
  const bool active = c < p.inner;
  float a[NPL], s[NPL], bv[NPL], cv[NPL];
#pragma unroll
  for (int i = 0; i < NPL; i++) a[i] = active && n0 + i < p.N ? p.a2[size_t(c) * p.N + n0 + i] : 0.f;
  const float d = active ? p.d[c] : 0.f;
  pdl::grid_dependency_wait();
  const int* seg = p.segs + 4 * blockIdx.y;
  const int row = seg[0], slot = seg[2];
  const bool fresh = p.positions[row] == 0;
  float* sp = p.ssm + (size_t(slot) * p.inner + c) * p.N + n0;
  const float* bc = p.bc + size_t(row) * p.ldbc + n0;
  const T* xz = static_cast<const T*>(p.xz);
  float u = 0.f, dt = 0.f, z = 0.f, roll = 0.f;
  // the convolution state moves up by one: lane k brings entry k + 1 (the last one: this token's input), all before any is stored
  const bool by_lanes = p.taps - 1 <= LPC, mine = active && by_lanes && lane < p.taps - 1;
  float* cs = p.conv_state + size_t(slot) * (p.taps - 1) * p.ldc + c;
  if (mine) roll = lane + 1 < p.taps - 1 ? cs[size_t(lane + 1) * p.ldc] : to_f(xz[size_t(row) * p.ldxz + c]);
  if (active) {
    u = to_f(static_cast<const T*>(p.u)[size_t(row) * p.ldu + c]);
    dt = p.dt[size_t(row) * p.lddt + c];
    z = to_f(xz[size_t(row) * p.ldxz + p.zoff + c]);
  }
#pragma unroll
  for (int i = 0; i < NPL; i++) {
    const bool ok = active && n0 + i < p.N;
    s[i] = ok ? sp[i] : 0.f;
    bv[i] = ok ? bc[p.boff + i] : 0.f;
    cv[i] = ok ? bc[p.coff + i] : 0.f;
  }
  dt = softplus<T>(dt);
  float y = 0.f;
#pragma unroll
  for (int i = 0; i < NPL; i++) {
    s[i] = fmaf(pow2<T>(dt * a[i]), fresh ? 0.f : s[i], dt * u * bv[i]);
    y = fmaf(s[i], cv[i], y);
    if (active && n0 + i < p.N) sp[i] = s[i];
  }
#pragma unroll
  for (int o = LPC / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (active && lane == 0) from_f(static_cast<T*>(p.out)[size_t(row) * p.ldo + c], fmaf(d, u, y) * gate<T>(z));
  __syncwarp();
  if (mine) cs[size_t(lane) * p.ldc] = fresh && lane + 1 < p.taps - 1 ? 0.f : roll;
  if (active && lane == 0 && !by_lanes) roll_conv_state(p, xz, row, 1, slot, fresh, c);
}

template <typename T, int LPC, int NPL>
cudaError_t launch_scan_t(const ScanParams& p, int nseg, bool one, cudaStream_t st) {
  const dim3 grid((p.inner + 128 / LPC - 1) / (128 / LPC), nseg);
  return one ? pdl::launch(k_scan_step<T, LPC, NPL>, grid, dim3(128), 0, st, 1, p) : pdl::launch(k_selective_scan<T, LPC, NPL>, grid, dim3(128), 0, st, 1, p);
}
template <typename T>
cudaError_t launch_scan(const ScanParams& p, int nseg, bool one, cudaStream_t st) {
  // few channels x segments: twice the lanes with half the states each keep more warps in flight
  const bool thin = !one && (long long)p.inner * nseg * 4 <= 148LL * 512;
  if (thin && p.N > 8 && p.N <= 16) return launch_scan_t<T, 8, 2>(p, nseg, one, st);
  if (p.N <= 4) return launch_scan_t<T, 1, 4>(p, nseg, one, st);
  if (p.N <= 8) return launch_scan_t<T, 2, 4>(p, nseg, one, st);
  if (p.N <= 16) return launch_scan_t<T, 4, 4>(p, nseg, one, st);
  if (p.N <= 32) return launch_scan_t<T, 8, 4>(p, nseg, one, st);
  if (p.N <= 64) return launch_scan_t<T, 16, 4>(p, nseg, one, st);
  if (p.N <= 128) return launch_scan_t<T, 32, 4>(p, nseg, one, st);
  return launch_scan_t<T, 32, 8>(p, nseg, one, st);
}
template <typename T>
cudaError_t launch_conv(const ConvParams& p, cudaStream_t st) {
  const int thr = p.ldc / 8 >= 128 ? 128 : ((p.ldc / 8 + 31) / 32) * 32;
  const int R = p.rows >= 512 ? 8 : 1;
  const dim3 grid((p.ldc / 8 + thr - 1) / thr, (p.rows + R - 1) / R);
  if (grid.y > 65535) return cudaErrorInvalidValue;
  auto go = [&](auto many, auto few) { return pdl::launch(R == 8 ? many : few, grid, dim3(thr), 0, st, 1, p); };
  switch (p.taps) {
    case 2: return go(k_causal_conv_silu<T, 2, 8>, k_causal_conv_silu<T, 2, 1>);
    case 3: return go(k_causal_conv_silu<T, 3, 8>, k_causal_conv_silu<T, 3, 1>);
    case 4: return go(k_causal_conv_silu<T, 4, 8>, k_causal_conv_silu<T, 4, 1>);
    default: return go(k_causal_conv_silu<T, 0, 8>, k_causal_conv_silu<T, 0, 1>);
  }
}

}  // namespace

extern "C" {

int tbv_op_causal_conv_silu(const void* x, void* out, const void* taps_w, const void* bias, const void* conv_state, const void* segs,
                            const void* seg_of_row, const void* positions, int rows, int ldx, int ldo, int ldc, int taps, int bf16,
                            void* stream) {
  if (rows <= 0) return 0;
  if ((ldc % 8) || (ldx % 8) || (ldo % 8) || taps < 1) return -2;
  ConvParams p{x, out, static_cast<const float*>(taps_w), static_cast<const float*>(bias), static_cast<const float*>(conv_state),
               static_cast<const int*>(segs), static_cast<const int*>(seg_of_row), static_cast<const int*>(positions),
               rows, ldx, ldo, ldc, taps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return (bf16 ? launch_conv<__nv_bfloat16>(p, st) : launch_conv<float>(p, st)) == cudaSuccess ? 0 : -1;
}

// one_token != 0: every segment has exactly one row
int tbv_op_selective_scan(const void* u, const void* xz, const void* dt, const void* bc, const void* a2, const void* d, void* ssm,
                          void* conv_state, void* out, const void* segs, const void* positions, int nseg, int inner, int N, int ldu,
                          int ldxz, int zoff, int lddt, int ldbc, int boff, int coff, int ldo, int ldc, int taps, int one_token, int bf16,
                          void* stream) {
  if (nseg <= 0) return 0;
  if (N < 1 || N > 256 || inner < 1 || taps < 1 || nseg > 65535) return -2;
  ScanParams p{u, xz, static_cast<const float*>(dt), static_cast<const float*>(bc), static_cast<const float*>(a2), static_cast<const float*>(d),
               static_cast<float*>(ssm), static_cast<float*>(conv_state), out, static_cast<const int*>(segs), static_cast<const int*>(positions),
               inner, N, ldu, ldxz, zoff, lddt, ldbc, boff, coff, ldo, ldc, taps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return (bf16 ? launch_scan<__nv_bfloat16>(p, nseg, one_token != 0, st) : launch_scan<float>(p, nseg, one_token != 0, st)) == cudaSuccess ? 0 : -1;
}

}  // extern "C"
