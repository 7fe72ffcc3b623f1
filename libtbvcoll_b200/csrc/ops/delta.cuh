// delta.cuh — parameters shared by the kernels of the gated delta rule with a decay per key channel (delta.cu, delta_chunk.cu).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "vec.cuh"

namespace delta_ops {

struct Params {
  const void *q, *k, *v;       // [rows, ld]: head g at g * Dp (q, k), head h at h * Vp (v); behind convolution and SiLU unless `taps_w` is given
  const void* beta;            // [rows, ldx]: logits, column h
  const void *low_a, *low_g;   // [rows, ldx]: what enters the second products of decays and gates (one-row form)
  const void *w_a, *b_a, *w_g; // [heads * Dp, rank], [heads * Dp], [heads * Vp, rank] (one-row form)
  const float* z;              // [rows, heads * Dp]: softplus of the decay inputs (many-row form)
  const void* gate;            // [rows, ldg]: gate logits (many-row form)
  const float* rate;           // [heads]: exp(A_log)
  const float* norm;           // [Vp]
  float* state;                // [slots, heads, Dp, Vp]
  float* o;                    // [rows, heads * Vp] scratch (many-row form)
  void* out;                   // [rows, ldo]
  const float* taps_w;         // one-row form: [taps, C] of the convolution over the C columns q | k | v, or null
  float* conv;                 // [slots, taps - 1, C]
  const int *segs, *positions;
  int heads, kv_heads, Dp, Vp, dim, vdim, ld, ldx, ldz, ldg, ldo, rank, taps, C;
  float eps;
};

constexpr float kUnitEps = 1e-6f;      // inside the root of the unit vectors' norm

// e^(-rate * s), s = softplus of the decay input: decay of one key channel
template <typename T> __device__ __forceinline__ float decay(float s, float rate);
template <> __device__ __forceinline__ float decay<float>(float s, float rate) { return expf(-rate * s); }
template <> __device__ __forceinline__ float decay<__nv_bfloat16>(float s, float rate) { return __expf(-rate * s); }

inline bool sizes_ok(const Params& p) {
  return p.heads > 0 && p.heads <= 65535 && p.kv_heads > 0 && p.heads % p.kv_heads == 0 && p.Dp > 0 && p.Dp <= 256 && p.Dp % 16 == 0 && p.Vp > 0 && p.Vp <= 1024 &&
         p.Vp % 16 == 0 && p.dim > 0 && p.dim <= p.Dp && p.vdim > 0 && p.vdim <= p.Vp;
}

// delta_chunk.cu: many rows of a bf16 model, in chunks on tensor cores; groups [ngroups, 4]: (first row, rows, state slot, -), together `rows` rows.  sets:
// null, or chunk_sets() bytes for the operands of all chunks (the form for few sequences and heads).  *finished: head norm and gate are done too (p.out),
// otherwise o is left in p.o.
bool chunk_fits(const Params& p);
size_t chunk_sets(const Params& p, int rows, int ngroups);
cudaError_t chunk_scan(const Params& p, const int* groups, int ngroups, int rows, void* sets, bool* finished, cudaStream_t st);

}  // namespace delta_ops
