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

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void from_f(float& d, float v) { d = v; }
__device__ __forceinline__ void from_f(__nv_bfloat16& d, float v) { d = __float2bfloat16_rn(v); }
__device__ __forceinline__ float silu(float v) { return v / (1.0f + __expf(-v)); }

__device__ __forceinline__ void load8(const float* p, float* f) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float* f) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
  f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
  f[4] = __uint_as_float(v.z << 16); f[5] = __uint_as_float(v.z & 0xffff0000u);
  f[6] = __uint_as_float(v.w << 16); f[7] = __uint_as_float(v.w & 0xffff0000u);
}
__device__ __forceinline__ void store8(float* p, const float* f) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float* f) {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; i++) {
    __nv_bfloat162 v = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
    w[i] = *reinterpret_cast<uint32_t*>(&v);
  }
  *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}

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

// out = silu(bias + sum_k w[k] * input at distance taps - 1 - k); a thread owns kConvRows consecutive rows of 8 channels
constexpr int kConvRows = 4;
template <typename T>
__global__ void __launch_bounds__(128) k_causal_conv_silu(const ConvParams p) {
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int c8 = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c8 >= p.ldc) return;
  const T* x = static_cast<const T*>(p.x);
  float bias[8];
  load8(p.bias + c8, bias);
  for (int r = 0; r < kConvRows; r++) {
    const int t = blockIdx.y * kConvRows + r;
    if (t >= p.rows) return;
    const int* sg = p.segs + 4 * (p.seg_of_row ? p.seg_of_row[t] : t);
    const int first = sg[0], j = t - first;
    const bool fresh = j >= p.taps - 1 ? true : p.positions[first] == 0;     // no carried input needed, or there is none
    float acc[8];
#pragma unroll
    for (int i = 0; i < 8; i++) acc[i] = bias[i];
    for (int k = 0; k < p.taps; k++) {
      const int back = p.taps - 1 - k;
      float v[8], w[8];
      if (back <= j) load8(x + size_t(t - back) * p.ldx + c8, v);
      else if (!fresh) load8(p.conv_state + (size_t(sg[2]) * (p.taps - 1) + (p.taps - 1 + j - back)) * p.ldc + c8, v);
      else continue;
      load8(p.taps_w + size_t(k) * p.ldc + c8, w);
#pragma unroll
      for (int i = 0; i < 8; i++) acc[i] = fmaf(w[i], v[i], acc[i]);
    }
#pragma unroll
    for (int i = 0; i < 8; i++) acc[i] = silu(acc[i]);
    store8(static_cast<T*>(p.out) + size_t(t) * p.ldo + c8, acc);
  }
}

struct ScanParams {
  const void* u;          // [rows, ldu]   convolved input
  const void* xz;         // [rows, ldxz]  convolution input (columns 0..) and gate (columns zoff ..)
  const float* dt;        // [rows, lddt]  step sizes, after the softplus
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

// LPC lanes share a channel, NPL states each (LPC * NPL >= N); a CTA owns 128 / LPC channels of one segment and walks its
// rows in tiles of TT: the tile's inputs are staged in shared memory while the next tile's are already on their way
// in registers.
template <typename T, int LPC, int NPL>
__global__ void __launch_bounds__(128) k_selective_scan(const ScanParams p) {
  constexpr int kC = 128 / LPC, NP = LPC * NPL;
  constexpr int TT = LPC == 1 ? 8 : (LPC == 2 ? 16 : (NP >= 128 ? 16 : 32));
  constexpr int EX = (TT * kC + 127) / 128, EB = (TT * NP + 127) / 128;
  __shared__ float su[TT][kC], sdt[TT][kC], sg[TT][kC], sy[TT][kC];
  __shared__ __align__(16) float sb[TT][NP];
  __shared__ __align__(16) float sc[TT][NP];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int* seg = p.segs + 4 * blockIdx.y;
  const int first = seg[0], count = seg[1], slot = seg[2];
  const bool fresh = p.positions[first] == 0;
  const int c0 = blockIdx.x * kC, cl = threadIdx.x / LPC, c = c0 + cl, lane = threadIdx.x % LPC, n0 = lane * NPL;
  const bool active = c < p.inner;
  const T* u = static_cast<const T*>(p.u);
  const T* xz = static_cast<const T*>(p.xz);
  T* out = static_cast<T*>(p.out);

  float a[NPL], s[NPL];
  float* sp = p.ssm + (size_t(slot) * p.inner + c) * p.N + n0;
#pragma unroll
  for (int i = 0; i < NPL; i++) {
    const bool ok = active && n0 + i < p.N;
    a[i] = ok ? p.a2[size_t(c) * p.N + n0 + i] : 0.f;
    s[i] = ok && !fresh ? sp[i] : 0.f;
  }
  const float dskip = active ? p.d[c] : 0.f;

  float ru[EX], rd[EX], rg[EX], rb[EB], rc[EB];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int e = 0; e < EX; e++) {
      const int id = threadIdx.x + e * 128, t = id / kC, cc = c0 + id % kC;
      const bool ok = id < TT * kC && t0 + t < count && cc < p.inner;
      const size_t row = size_t(first) + t0 + t;
      ru[e] = ok ? to_f(u[row * p.ldu + cc]) : 0.f;
      rd[e] = ok ? p.dt[row * p.lddt + cc] : 0.f;
      rg[e] = ok ? to_f(xz[row * p.ldxz + p.zoff + cc]) : 0.f;
    }
#pragma unroll
    for (int e = 0; e < EB; e++) {
      const int id = threadIdx.x + e * 128, t = id / NP, n = id % NP;
      const bool ok = id < TT * NP && t0 + t < count && n < p.N;
      const size_t row = size_t(first) + t0 + t;
      rb[e] = ok ? p.bc[row * p.ldbc + p.boff + n] : 0.f;
      rc[e] = ok ? p.bc[row * p.ldbc + p.coff + n] : 0.f;
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < count; t0 += TT) {
    const int nt = min(TT, count - t0);
    __syncthreads();
#pragma unroll
    for (int e = 0; e < EX; e++) {
      const int id = threadIdx.x + e * 128;
      if (id < TT * kC) {
        su[id / kC][id % kC] = ru[e];
        sdt[id / kC][id % kC] = rd[e];
        sg[id / kC][id % kC] = silu(rg[e]);
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
#pragma unroll 4
    for (int t = 0; t < nt; t++) {
      const float dt = sdt[t][cl], x = su[t][cl], dx = dt * x;
      float y = 0.f;
#pragma unroll
      for (int i = 0; i < NPL; i++) {
        s[i] = fmaf(exp2f(dt * a[i]), s[i], dx * sb[t][n0 + i]);
        y = fmaf(s[i], sc[t][n0 + i], y);
      }
#pragma unroll
      for (int o = LPC / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (lane == 0) sy[t][cl] = fmaf(dskip, x, y);
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < EX; e++) {
      const int id = threadIdx.x + e * 128, t = id / kC, cc = id % kC;
      if (id < TT * kC && t < nt && c0 + cc < p.inner) from_f(out[(size_t(first) + t0 + t) * p.ldo + c0 + cc], sy[t][cc] * sg[t][cc]);
    }
  }
#pragma unroll
  for (int i = 0; i < NPL; i++)
    if (active && n0 + i < p.N) sp[i] = s[i];
  // the convolution's last taps - 1 inputs; ascending, so an old entry is read before it is overwritten
  if (active && lane == 0) {
    float* cs = p.conv_state + size_t(slot) * (p.taps - 1) * p.ldc + c;
    for (int k = 0; k < p.taps - 1; k++) {
      const int j = count - (p.taps - 1) + k;
      cs[size_t(k) * p.ldc] = j >= 0 ? to_f(xz[(size_t(first) + j) * p.ldxz + c]) : (fresh ? 0.f : cs[size_t(k + count) * p.ldc]);
    }
  }
}

template <typename T>
cudaError_t launch_scan(const ScanParams& p, int nseg, cudaStream_t st) {
  auto go = [&](auto kern, int lpc) { return pdl::launch(kern, dim3((p.inner + 128 / lpc - 1) / (128 / lpc), nseg), dim3(128), 0, st, 1, p); };
  if (p.N <= 4) return go(k_selective_scan<T, 1, 4>, 1);
  if (p.N <= 8) return go(k_selective_scan<T, 2, 4>, 2);
  if (p.N <= 16) return go(k_selective_scan<T, 4, 4>, 4);
  if (p.N <= 32) return go(k_selective_scan<T, 8, 4>, 8);
  if (p.N <= 64) return go(k_selective_scan<T, 16, 4>, 16);
  if (p.N <= 128) return go(k_selective_scan<T, 32, 4>, 32);
  return go(k_selective_scan<T, 32, 8>, 32);
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
  const int thr = ldc / 8 >= 128 ? 128 : ((ldc / 8 + 31) / 32) * 32;
  const dim3 grid((ldc / 8 + thr - 1) / thr, (rows + kConvRows - 1) / kConvRows);
  if (grid.y > 65535) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = bf16 ? pdl::launch(k_causal_conv_silu<__nv_bfloat16>, grid, dim3(thr), 0, st, 1, p)
                       : pdl::launch(k_causal_conv_silu<float>, grid, dim3(thr), 0, st, 1, p);
  return e == cudaSuccess ? 0 : -1;
}

int tbv_op_selective_scan(const void* u, const void* xz, const void* dt, const void* bc, const void* a2, const void* d, void* ssm,
                          void* conv_state, void* out, const void* segs, const void* positions, int nseg, int inner, int N, int ldu,
                          int ldxz, int zoff, int lddt, int ldbc, int boff, int coff, int ldo, int ldc, int taps, int bf16, void* stream) {
  if (nseg <= 0) return 0;
  if (N < 1 || N > 256 || inner < 1 || taps < 1 || nseg > 65535) return -2;
  ScanParams p{u, xz, static_cast<const float*>(dt), static_cast<const float*>(bc), static_cast<const float*>(a2), static_cast<const float*>(d),
               static_cast<float*>(ssm), static_cast<float*>(conv_state), out, static_cast<const int*>(segs), static_cast<const int*>(positions),
               inner, N, ldu, ldxz, zoff, lddt, ldbc, boff, coff, ldo, ldc, taps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return (bf16 ? launch_scan<__nv_bfloat16>(p, nseg, st) : launch_scan<float>(p, nseg, st)) == cudaSuccess ? 0 : -1;
}

}  // extern "C"
