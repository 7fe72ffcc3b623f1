// moe.cu — routing of a mixture of experts: scores = softmax of the router's logits over all experts, the `top` largest chosen (the lower index of
// equal ones), their scores divided by their sum and scaled.  The chosen (token, expert) pairs are laid out expert after expert; a
// token's row is copied to each of its places, so that the experts' products (row-grouped GEMM) read and write consecutive rows.
//
//   place [T, top]   row of the j-th choice in the permuted arrays        offsets [E + 1]   first row of every expert
//   weight [T, top]
//
// Up to kSmall tokens: one kernel, in which every CTA routes all tokens and moves one.  More: k_route (a warp per token; ranks from atomic
// counters, so that the order inside an expert is not fixed — no row's result depends on it), then k_dispatch.
//
// Where the choice is looked up by token id instead, places depend on the ids alone: one launch lays out all such layers of a model at the start of a step
// (k_place_table, a CTA per layer), and whoever makes the rows writes them to their places.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../pdl.cuh"

namespace {

constexpr int kSmall = 32, kMaxExperts = 512, kMaxTop = 64;

struct RouteParams {
  const float* logits;    // [T, lde]
  int T, E, lde, top;
  float scale;
  const void* h;          // [T, row_bytes]
  void* xp;               // [T * top, row_bytes]
  int *place, *offsets, *counts;
  float* weight;
  int* choice;            // [T, 2 * top]: expert, rank (large form)
  int units;              // 16-byte units of a row
};

// One warp: the chosen experts of logits z go to idx[0..top), their weights to w[0..top) (either may be null).  `sc` = E floats of shared memory.
__device__ __forceinline__ void choose(const float* z, int E, int top, float scale, float* sc, int* idx, float* w) {
  const int lane = threadIdx.x & 31;
  float m = -INFINITY;
  for (int e = lane; e < E; e += 32) { const float v = z[e]; sc[e] = v; m = fmaxf(m, v); }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
  float l = 0.f;
  for (int e = lane; e < E; e += 32) { const float v = expf(sc[e] - m); sc[e] = v; l += v; }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
  float sum = 0.f;
  for (int j = 0; j < top; j++) {
    float best = -1.f;
    int at = E;
    for (int e = lane; e < E; e += 32)
      if (sc[e] > best) { best = sc[e]; at = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
    }
    at = min(at, E - 1);                 // logits that are not numbers compare with nothing: stay inside
    const float s = best / l;
    sum += s;
    if (lane == 0) {
      if (idx) idx[j] = at;
      if (w) w[j] = s;
    }
    if (lane == (at & 31)) sc[at] = -1.f;
    __syncwarp();
  }
  if (w && lane == 0)
    for (int j = 0; j < top; j++) w[j] = w[j] / (sum + 1e-20f) * scale;
}

// exclusive prefix sums of n values (shared memory), by one warp; out[n] = total
__device__ __forceinline__ void warp_prefix(const int* in, int* out, int n) {
  const int lane = threadIdx.x & 31, per = (n + 31) / 32, a = min(n, lane * per), b = min(n, a + per);
  int s = 0;
  for (int i = a; i < b; i++) s += in[i];
  int inc = s;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc += v;
  }
  int run = inc - s;
  for (int i = a; i < b; i++) { out[i] = run; run += in[i]; }
  if (lane == 31) out[n] = inc;
}

__global__ void __launch_bounds__(256) k_route_small(const RouteParams p) {
  extern __shared__ int sm[];
  int* idx = sm;                                   // [T][top]
  int* cnt = idx + p.T * p.top;                    // [E]
  int* off = cnt + p.E;                            // [E + 1]
  float* sc = reinterpret_cast<float*>(off + p.E + 1);   // [8][E]
  __shared__ int place[kMaxTop];
  pdl::launch_dependents();
  for (int e = threadIdx.x; e < p.E; e += 256) cnt[e] = 0;
  pdl::grid_dependency_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, own = blockIdx.x;
  for (int t = warp; t < p.T; t += 8)
    choose(p.logits + size_t(t) * p.lde, p.E, p.top, p.scale, sc + warp * p.E, idx + t * p.top, t == own ? p.weight + size_t(t) * p.top : nullptr);
  __syncthreads();
  for (int i = threadIdx.x; i < p.T * p.top; i += 256) atomicAdd(&cnt[idx[i]], 1);
  __syncthreads();
  if (warp == 0) warp_prefix(cnt, off, p.E);
  __syncthreads();
  for (int j = warp; j < p.top; j += 8) {
    const int e = idx[own * p.top + j];
    int before = 0;
    for (int i = lane; i < own * p.top; i += 32) before += idx[i] == e;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
    if (lane == 0) {
      place[j] = off[e] + before;
      p.place[own * p.top + j] = place[j];
    }
  }
  if (own == 0)
    for (int e = threadIdx.x; e <= p.E; e += 256) p.offsets[e] = off[e];
  __syncthreads();
  const uint4* src = static_cast<const uint4*>(p.h) + size_t(own) * p.units;
  for (int i = threadIdx.x; i < p.units; i += 256) {
    const uint4 v = src[i];
    for (int j = 0; j < p.top; j++) static_cast<uint4*>(p.xp)[size_t(place[j]) * p.units + i] = v;
  }
}

__global__ void __launch_bounds__(256) k_route(const RouteParams p) {
  extern __shared__ float scs[];                   // [8][E]
  __shared__ int idx[8][kMaxTop];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 8 + warp;
  if (t >= p.T) return;
  choose(p.logits + size_t(t) * p.lde, p.E, p.top, p.scale, scs + warp * p.E, idx[warp], p.weight + size_t(t) * p.top);
  __syncwarp();
  for (int j = lane; j < p.top; j += 32) {
    const int e = idx[warp][j];
    p.choice[(size_t(t) * p.top + j) * 2] = e;
    p.choice[(size_t(t) * p.top + j) * 2 + 1] = atomicAdd(&p.counts[e], 1);
  }
}

__global__ void __launch_bounds__(256) k_dispatch(const RouteParams p) {
  __shared__ int cnt[kMaxExperts], off[kMaxExperts + 1];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  for (int e = threadIdx.x; e < p.E; e += 256) cnt[e] = p.counts[e];
  __syncthreads();
  if (threadIdx.x < 32) warp_prefix(cnt, off, p.E);
  __syncthreads();
  if (blockIdx.x == 0)
    for (int e = threadIdx.x; e <= p.E; e += 256) p.offsets[e] = off[e];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 8 + warp;
  if (t >= p.T) return;
  const int* ch = p.choice + size_t(t) * p.top * 2;
  for (int j = lane; j < p.top; j += 32) p.place[t * p.top + j] = off[ch[2 * j]] + ch[2 * j + 1];
  const uint4* src = static_cast<const uint4*>(p.h) + size_t(t) * p.units;
  for (int i = lane; i < p.units; i += 128) {      // four units per lane in flight
    uint4 v[4];
#pragma unroll
    for (int k = 0; k < 4; k++)
      if (i + 32 * k < p.units) v[k] = src[i + 32 * k];
    for (int j = 0; j < p.top; j++) {
      uint4* dst = static_cast<uint4*>(p.xp) + size_t(off[ch[2 * j]] + ch[2 * j + 1]) * p.units + i;
#pragma unroll
      for (int k = 0; k < 4; k++)
        if (i + 32 * k < p.units) dst[32 * k] = v[k];
    }
  }
}

// One layer's table and results; as laid out in device memory by the caller.
struct TableLayer {
  const int* table;      // [vocab, top]: the experts of every token id, all different
  int* place;            // [T, top]
  int* offsets;          // [E + 1]
  int E, top;
};

__global__ void __launch_bounds__(1024) k_place_table(const long long* __restrict__ ids, const TableLayer* __restrict__ layers, int T, long long vocab) {
  __shared__ int cnt[kMaxExperts], off[kMaxExperts + 1];
  pdl::launch_dependents();
  const TableLayer l = layers[blockIdx.x];
  for (int e = threadIdx.x; e < l.E; e += 1024) cnt[e] = 0;
  __syncthreads();
  pdl::grid_dependency_wait();
  const int n = T * l.top;
  auto expert = [&](int i) {
    const long long id = ids[i / l.top];
    const int e = l.table[size_t(id < 0 ? 0 : (id >= vocab ? vocab - 1 : id)) * l.top + i % l.top];
    return e < 0 ? 0 : (e >= l.E ? l.E - 1 : e);
  };
  for (int i = threadIdx.x; i < n; i += 1024) l.place[i] = atomicAdd(&cnt[expert(i)], 1);
  __syncthreads();
  if (threadIdx.x < 32) warp_prefix(cnt, off, l.E);
  __syncthreads();
  for (int e = threadIdx.x; e <= l.E; e += 1024) l.offsets[e] = off[e];
  for (int i = threadIdx.x; i < n; i += 1024) l.place[i] += off[expert(i)];
}

}  // namespace

extern "C" {

int tbv_op_moe_small(void) { return kSmall; }

// logits fp32 [T, lde]; h, xp: rows of row_bytes (a multiple of 16).  counts [E] and choice [T, 2 top] (ints) are scratch of the many-token form.
int tbv_op_moe_route(const void* logits, const void* h, void* xp, void* place, void* weight, void* offsets, void* counts, void* choice, int T,
                     int E, int lde, int top, float scale, int row_bytes, void* stream) {
  if (T <= 0) return 0;
  if (E < 1 || E > kMaxExperts || top < 1 || top > E || top > kMaxTop || lde < E || (row_bytes % 16)) return -2;
  RouteParams p{static_cast<const float*>(logits), T, E, lde, top, scale, h, xp, static_cast<int*>(place), static_cast<int*>(offsets),
                static_cast<int*>(counts), static_cast<float*>(weight), static_cast<int*>(choice), row_bytes / 16};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (T <= kSmall) {
    const size_t smem = (size_t(T) * top + 2 * E + 1 + 8 * E) * 4;      // at most 29 KB
    e = pdl::launch(k_route_small, dim3(T), dim3(256), smem, st, 1, p);
  } else {
    if (cudaMemsetAsync(counts, 0, size_t(E) * 4, st) != cudaSuccess) return -1;
    e = pdl::launch(k_route, dim3((T + 7) / 8), dim3(256), size_t(8) * E * 4, st, 1, p);
    if (e == cudaSuccess) e = pdl::launch(k_dispatch, dim3((T + 7) / 8), dim3(256), 0, st, 1, p);
  }
  return e == cudaSuccess ? 0 : -1;
}

// Places and offsets of `nlayers` layers whose experts come from tables (TableLayer records in device memory: three pointers, experts, top; at most
// max_experts experts).  ids int64 [T].
int tbv_op_moe_place_table(const void* ids, const void* layers, int nlayers, int max_experts, int T, long long vocab, void* stream) {
  if (T <= 0 || nlayers <= 0) return 0;
  if (max_experts < 1 || max_experts > kMaxExperts || vocab < 1) return -2;
  return pdl::launch(k_place_table, dim3(nlayers), dim3(1024), 0, static_cast<cudaStream_t>(stream), 1, static_cast<const long long*>(ids),
                     static_cast<const TableLayer*>(layers), T, vocab) == cudaSuccess ? 0 : -1;
}

}  // extern "C"
