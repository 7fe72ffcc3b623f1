// decay.cuh — parameters and decays shared by the kernels of linear recurrences with a matrix state (decay_scan.cu, chunk_scan.cu, fixed_decay.cu).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace decay_ops {

struct ScanParams {
  const void *q, *k, *v, *g;   // [rows, ld]: column h * Dp (q, k) or h * Vp (v, g) of each pointer
  const float* z;              // [rows, ldz] decay inputs (many rows)
  const void *low, *w2, *b2;   // or z = low . w2 + b2, low [rows, ldlow], w2 [heads * Dp, rank], b2 [heads * Dp]
  const float* u;              // [heads * Dp]: WKV (null: gated linear attention)
  const float* norm;           // [heads * Vp]
  float* state;
  float* o;                    // [rows, heads * Vp] (many rows)
  void* out;                   // [rows, ldo]
  const float* h1;             // [rows, ldh] inputs whose last row per segment goes to shift [slots, ldh] (null: none)
  float* shift;
  const int *segs, *positions;
  int heads, Dp, Vp, vdim, ld, ldz, ldlow, rank, ldo, ldh;
  float qscale, inv_tau, eps;
  const float* fixed;          // one constant decay per head instead of z, at fixed[h * fixed_ld] (32-bit sequential kernel only)
  int fixed_ld;
};

// decay of one key channel; bf16 models take the fast exponential and logarithm (1 + e^-|z| lies in 1 .. 2: absolute error about 1e-7)
template <typename T> __device__ __forceinline__ float decay(float z, bool wkv, float inv_tau);
template <> __device__ __forceinline__ float decay<float>(float z, bool wkv, float inv_tau) {
  if (wkv) return expf(-expf(z));
  return expf(-(fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))) * inv_tau);
}
template <> __device__ __forceinline__ float decay<__nv_bfloat16>(float z, bool wkv, float inv_tau) {
  if (wkv) return __expf(-__expf(z));
  return __expf(-(fmaxf(-z, 0.f) + __logf(1.f + __expf(-fabsf(z)))) * inv_tau);
}

inline bool sizes_ok(int heads, int Dp, int Vp) { return heads > 0 && heads <= 65535 && Dp > 0 && Dp <= 256 && (Dp % 16) == 0 && Vp > 0 && Vp <= 1024 && (Vp % 16) == 0; }

// decay_scan.cu: q, k, v and decays -> o (p.o), token by token in fp32
cudaError_t sequential_scan_f32(const ScanParams& p, int nseg, cudaStream_t st);
// chunk_scan.cu: the recurrence of a bf16 model over many rows.  groups [ngroups, 4]: (first row, rows, state slot, flags: 1 = a group of the same
// segment precedes, 2 = one follows).  p.z null: decay inputs from p.low, p.w2, p.b2 (p.low as it enters the product).  *finished: head norm and gate
// are done too (p.out), otherwise o is left in p.o.
constexpr int kMaxRank = 128;     // of the fused decay product
cudaError_t chunk_scan(const ScanParams& p, const int* groups, int ngroups, bool multi, float* starts, float* totals, bool* finished, cudaStream_t st);

}  // namespace decay_ops
