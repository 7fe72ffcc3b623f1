// short_conv.cu — short causal convolution over time, one filter per channel, over ragged batches with carried state:
//
//   y_t = act(sum_j w[j] x_{t - taps + 1 + j})            or, added to its input,   y_t = x_t + sum_j w[j] x_{t - taps + 1 + j}
//
// Rows of a sequence are consecutive (segments as in mamba.cu); zeros stand before a sequence's start, the carried inputs before a portion's.
// State fp32 [slots, taps - 1, C]: the last taps - 1 inputs, oldest first.  The first taps - 1 rows of a segment need the state and the last ones replace
// it; one thread does both for its channels, so that no other launch is needed.  All other rows see rows of the batch only.
//
// The one-row-per-segment forms lie in the kernels that make the input (residual.cu) or use the result (delta.cu).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../pdl.cuh"
#include "vec.cuh"

namespace {

using namespace vec;

struct ShortConvParams {
  const void* x;             // [rows, ldx]
  void* out;                 // [rows, ldo]
  const float* taps_w;       // [taps, C], row taps - 1 weighs the current token
  float* state;              // [slots, taps - 1, C]
  const int* segs;           // [nseg, 4]
  const int* seg_of_row;     // [rows] or null (row i = segment i)
  const int* positions;      // [rows]
  int rows, ldx, ldo, C, taps;
};

// A thread owns R consecutive rows of 8 channels; TAPS 0: any number.
template <typename TI, typename TO, bool ADD, int TAPS, int R>
__global__ void __launch_bounds__(128) k_short_conv(const ShortConvParams p) {
  pdl::launch_dependents();
  const int c8 = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  const int taps = TAPS > 0 ? TAPS : p.taps;
  float w[TAPS > 0 ? TAPS : 1][8];
  if (TAPS > 0 && c8 < p.C) {                // weights: no need to wait for the kernel before
#pragma unroll
    for (int k = 0; k < TAPS; k++) load8(p.taps_w + size_t(k) * p.C + c8, w[k]);
  }
  pdl::grid_dependency_wait();
  if (c8 >= p.C) return;
  const TI* x = static_cast<const TI*>(p.x) + c8;
  TO* out = static_cast<TO*>(p.out) + c8;
  auto put = [&](int t, float* acc, const float* own) {
#pragma unroll
    for (int i = 0; i < 8; i++) acc[i] = ADD ? own[i] + acc[i] : gate<TO>(acc[i]);
    store8(out + size_t(t) * p.ldo, acc);
  };
  auto tap = [&](int k, const float* v, float* acc) {
    float wk[8];
    if (TAPS == 0) load8(p.taps_w + size_t(k) * p.C + c8, wk);
#pragma unroll
    for (int i = 0; i < 8; i++) acc[i] = fmaf(TAPS > 0 ? w[TAPS > 0 ? k : 0][i] : wk[i], v[i], acc[i]);
  };
  const int t0 = blockIdx.y * R;
  if (R > 1 && TAPS > 0 && t0 >= TAPS - 1 && t0 + R <= p.rows) {
    // the window is requested before it is known whether the rows share a segment
    Raw8<TI> win[TAPS > 0 ? TAPS + R - 1 : 1];
#pragma unroll
    for (int i = 0; i < TAPS + R - 1; i++) win[i].load(x + size_t(t0 - (TAPS - 1) + i) * p.ldx);
    const int sa = p.seg_of_row ? p.seg_of_row[t0] : t0, sb = p.seg_of_row ? p.seg_of_row[t0 + R - 1] : t0 + R - 1;
    if (sa == sb && t0 - p.segs[4 * sa] >= TAPS - 1) {
#pragma unroll
      for (int r = 0; r < R; r++) {
        float acc[8] = {}, v[8];
#pragma unroll
        for (int k = 0; k < TAPS; k++) {
          win[r + k].unpack(v);
          tap(k, v, acc);
        }
        put(t0 + r, acc, v);                  // the last input taken is the row's own
      }
      return;
    }
  }
  for (int r = 0; r < R; r++) {
    const int t = t0 + r;
    if (t >= p.rows) return;
    const int* sg = p.segs + 4 * (p.seg_of_row ? p.seg_of_row[t] : t);
    const int first = sg[0], n = sg[1], j = t - first, keep = taps - 1;
    if (j > 0 && j < keep) continue;          // done with the segment's first row
    if (j >= keep) {
      float acc[8] = {}, v[8] = {};
      for (int k = 0; k < taps; k++) {
        load8(x + size_t(t - keep + k) * p.ldx, v);
        tap(k, v, acc);
      }
      put(t, acc, v);
      continue;
    }
    const bool fresh = p.positions[first] == 0;
    float* st = p.state + size_t(sg[2]) * keep * p.C + c8;
    auto input = [&](int i, float* v) {       // input i of the segment; before it: carried inputs, or zeros
      if (i >= 0) load8(x + size_t(first + i) * p.ldx, v);
      else if (!fresh) load8(st + size_t(keep + i) * p.C, v);
      else {
#pragma unroll
        for (int e = 0; e < 8; e++) v[e] = 0.f;
      }
    };
    const int heads = keep > 0 ? min(n, keep) : 1;
    for (int i = 0; i < heads; i++) {
      float acc[8] = {}, v[8];
      for (int k = 0; k < taps; k++) {
        input(i - keep + k, v);
        tap(k, v, acc);
      }
      put(first + i, acc, v);
    }
    for (int i = 0; i < keep; i++) {          // ascending: an old entry is read before it is overwritten
      float v[8];
      input(n - keep + i, v);
      store8(st + size_t(i) * p.C, v);
    }
  }
}

template <typename TI, typename TO, bool ADD>
cudaError_t launch(const ShortConvParams& p, cudaStream_t st) {
  const int units = (p.C + 7) / 8, threads = units < 128 ? (units + 31) / 32 * 32 : 128;
  constexpr int R = 4;
  const bool few = p.rows <= 64;
  const dim3 grid((units + threads - 1) / threads, few ? p.rows : (p.rows + R - 1) / R), blk(threads);
  if (few) return pdl::launch(k_short_conv<TI, TO, ADD, 0, 1>, grid, blk, 0, st, 1, p);
  switch (p.taps) {
    case 2: return pdl::launch(k_short_conv<TI, TO, ADD, 2, R>, grid, blk, 0, st, 1, p);
    case 3: return pdl::launch(k_short_conv<TI, TO, ADD, 3, R>, grid, blk, 0, st, 1, p);
    case 4: return pdl::launch(k_short_conv<TI, TO, ADD, 4, R>, grid, blk, 0, st, 1, p);
    default: return pdl::launch(k_short_conv<TI, TO, ADD, 0, R>, grid, blk, 0, st, 1, p);
  }
}

}  // namespace

extern "C" {

// add: out = x + conv(x), x fp32 and out in the activation type; otherwise out = silu(conv(x)), both in the activation type.
int tbv_op_short_conv(const void* x, void* out, const void* taps_w, void* state, const void* segs, const void* seg_of_row, const void* positions, int rows,
                      int ldx, int ldo, int C, int taps, int add, int bf16, void* stream) {
  if (rows <= 0) return 0;
  if (C <= 0 || (C % 8) || (ldx % 8) || (ldo % 8) || ldx < C || ldo < C || taps < 1 || !segs || !positions || (taps > 1 && !state)) return -2;
  ShortConvParams p{x, out, static_cast<const float*>(taps_w), static_cast<float*>(state), static_cast<const int*>(segs),
                    static_cast<const int*>(seg_of_row), static_cast<const int*>(positions), rows, ldx, ldo, C, taps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (add) e = bf16 ? launch<float, __nv_bfloat16, true>(p, st) : launch<float, float, true>(p, st);
  else e = bf16 ? launch<__nv_bfloat16, __nv_bfloat16, false>(p, st) : launch<float, float, false>(p, st);
  return e == cudaSuccess ? 0 : -1;
}

}  // extern "C"
