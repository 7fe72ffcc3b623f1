// residual.cu — one fp32 residual stream with parallel branches: what lies between two layers in one kernel.
//
// A layer is x <- x + mixer(norm1(x)) + ff(norm2(x)).  The kernel that ends it adds the branches' results and starts the next layer:
//   x  <- x + y1 + y2 + sum_j weight_j * routed[place_j]        (each term optional; the last is a mixture of experts)
//   x  <- x + x0 + step                                           (optional: a loop's pass begins; x0 is the stream as the embedding left it)
//   h1 = norm(x) * gamma1,  h2 = norm(x) * gamma2                 (both norms are of the same x: one root mean square)
// or, for the embedding, x = table[id] * scale + position vector.  Sine and cosine come from turns = position * frequency / 2 pi in two
// fp32 pieces, reduced before they are rounded.  For layers that mix every token with the one before, h1 stays fp32; when every
// sequence has one row (a decode step) the mixes are written here, with the previous token's h1 from the carried state; otherwise
// k_token_shift writes them from h1.
//
// Layers with a norm before and behind every sublayer, x <- x + norm_b(f(norm_a(x))), use the same kernel with a second reduction (POST): the
// branches' sum goes through a norm of its own before it is added.  If what entered the branch's last product was still to be divided by a root mean
// square of its row (the joint norm of a recurrence's heads), its square sums come along (`sums`) and the product is divided here.  h1 may
// go straight to the rows of a row-grouped product (`out_place`) instead of to its own row.
//
// Layers with the norm behind the sublayer only take h1 = x (no gamma1), and a short causal convolution of the stream may be added to it: h1 = x + conv(x).
// When every sequence has one row that happens here, with the inputs before it from the carried state, which is replaced (`near`); otherwise
// short_conv.cu makes h1 and this kernel leaves it out (no h1).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../pdl.cuh"
#include "vec.cuh"

using vec::sincos_turns;

namespace {

constexpr int kThreads = 512;
constexpr int kMaxUnits = 16;       // float4 units of a row per thread: width <= 512 * 16 * 4
constexpr int kMaxTop = 64;
constexpr int kNear = 3;            // carried inputs of the convolution taken at once

struct ResidualParams {
  // embedding
  const long long* ids;
  const void* table;                // [vocab, ld] in the activation type
  const float2* freq;               // [ceil(width / 2)]: turns per position, high and low part (null: no position vector)
  const int* positions;
  float embed_scale;
  long long vocab;
  // branches
  float* x;                         // [rows, ld]
  float* x0;                        // embedding: stored if given; otherwise added if given
  const float *y1, *y2, *step;      // [rows, ld], [rows, ld], [ld]
  const void* routed;               // [places, ld] in the activation type
  const int* place;                 // [rows, top]
  const float* weight;              // [rows, top]; null: every weight is `weight_const`
  float weight_const;
  int top;
  const float* post;                // POST: [ld] weight of the branches' norm
  const float* sums;                // POST: [rows, nsum] square sums, or null: the branches are divided by sqrt(their sum / sum_width + eps)
  int nsum, sum_width;
  // norms
  const float *g1, *g2;
  void *h1, *h2;                    // [rows, ldh]
  const int* out_place;             // [rows, out_top]: h1 goes to these rows (null: to its own)
  int out_top;
  int h1_f32;
  const long long* rows;            // last: source row of every output row (null = identity); x is not written
  int last;
  // mixes with the previous token (one row per sequence)
  const float* mu;                  // [nmix, ld]
  void* mixes;                      // [rows, nmix, ld]
  float* shift;                     // [slots, ld]
  const int* segs;
  int nmix;
  // h1 += conv(h1) over time (one row per sequence); state of the last `taps` - 1 inputs
  const float* near;                // [taps, ld], the last row weighs the current token
  float* past;                      // [slots, taps - 1, ld]
  int taps;
  int width, ld, ldh;
  float eps;
};

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}
__device__ __forceinline__ void add4(float4& a, const float4& b) { a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w; }
__device__ __forceinline__ void fma4(float4& a, float s, const float4& b) { a.x = fmaf(s, b.x, a.x); a.y = fmaf(s, b.y, a.y); a.z = fmaf(s, b.z, a.z); a.w = fmaf(s, b.w, a.w); }
__device__ __forceinline__ void mul_add4(float4& a, const float4& s, const float4& b) {
  a.x = fmaf(s.x, b.x, a.x); a.y = fmaf(s.y, b.y, a.y); a.z = fmaf(s.z, b.z, a.z); a.w = fmaf(s.w, b.w, a.w);
}
__device__ __forceinline__ float4 mix4(const float4& h, const float4& prev, const float4& mu) {
  return make_float4(fmaf(prev.x - h.x, mu.x, h.x), fmaf(prev.y - h.y, mu.y, h.y), fmaf(prev.z - h.z, mu.z, h.z), fmaf(prev.w - h.w, mu.w, h.w));
}
// Sums over the block of at most 16 warps: warp_part before a barrier, block_total behind it (in every thread).
__device__ __forceinline__ void warp_part(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
}
__device__ __forceinline__ float block_total(const float* red) {
  const int w = threadIdx.x & 15;
  float v = w < int(blockDim.x) / 32 ? red[w] : 0.f;
#pragma unroll
  for (int o = 8; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// NEAR: with the convolution (an instance of its own: it holds more registers)
template <typename T, bool EMBED, bool POST, bool NEAR, int U>
__global__ void __launch_bounds__(kThreads) k_residual(const ResidualParams p) {
  __shared__ float red[16], red_b[16], red_s[16], sw[kMaxTop];
  __shared__ int sp[kMaxTop], so[kMaxTop];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int units = p.ld / 4;
  const size_t row = p.last && p.rows ? size_t(p.rows[blockIdx.x]) : blockIdx.x;
  if (p.out_place && threadIdx.x < p.out_top) so[threadIdx.x] = p.out_place[row * p.out_top + threadIdx.x];   // read behind a reduction's barrier
  if (!EMBED && p.routed) {
    if (threadIdx.x < p.top) {
      sp[threadIdx.x] = p.place[row * p.top + threadIdx.x];
      sw[threadIdx.x] = p.weight ? p.weight[row * p.top + threadIdx.x] : p.weight_const;
    }
    __syncthreads();
  }
  float* xr = p.x + row * p.ld;
  // carried inputs of the convolution: requested here where registers allow, long before they are used
  constexpr bool kEarly = NEAR && U <= 2;
  float4 pre[kEarly ? U : 1][kNear];
  float* past = nullptr;
  bool fresh = true;
  if constexpr (NEAR) {
    past = p.past + size_t(p.segs[4 * blockIdx.x + 2]) * (p.taps - 1) * p.ld;
    fresh = p.positions[row] == 0;
    if (kEarly) {
#pragma unroll
      for (int k = 0; k < U; k++)
#pragma unroll
        for (int j = 0; j < kNear; j++) {
          const int i = threadIdx.x + k * blockDim.x;
          pre[kEarly ? k : 0][j] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (i < units && j < p.taps - 1 && !fresh) pre[kEarly ? k : 0][j] = load4(past + size_t(j) * p.ld + i * 4);
        }
    }
  }
  float4 u[U], b[POST ? U : 1];
  if constexpr (POST) {
    float sb = 0.f, sq = 0.f;
    if (p.sums)
      for (int i = threadIdx.x; i < p.nsum; i += blockDim.x) sq += p.sums[row * p.nsum + i];
#pragma unroll
    for (int k = 0; k < U; k++) {
      const int i = threadIdx.x + k * blockDim.x;
      b[k] = u[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < units) {
        u[k] = load4(xr + i * 4);
        if (p.y1) b[k] = load4(p.y1 + row * p.ld + i * 4);
        if (p.routed) {
          const T* ro = static_cast<const T*>(p.routed) + i * 4;
#pragma unroll 4
          for (int j = 0; j < p.top; j++) fma4(b[k], sw[j], load4(ro + size_t(sp[j]) * p.ld));
        }
        sb += b[k].x * b[k].x + b[k].y * b[k].y + b[k].z * b[k].z + b[k].w * b[k].w;
      }
    }
    warp_part(sb, red_b);
    if (p.sums) warp_part(sq, red_s);
    __syncthreads();
    float f = p.sums ? 1.0f / sqrtf(block_total(red_s) / float(p.sum_width) + p.eps) : 1.0f;
    f /= sqrtf(block_total(red_b) * f * f / float(p.width) + p.eps);
#pragma unroll
    for (int k = 0; k < U; k++) {
      const int i = threadIdx.x + k * blockDim.x;
      if (i < units) {
        const float4 g = load4(p.post + i * 4);
        b[k] = make_float4(b[k].x * f * g.x, b[k].y * f * g.y, b[k].z * f * g.z, b[k].w * f * g.w);
      }
    }
  }
  float ss = 0.f;
  const T* erow = nullptr;
  float pos = 0.f;
  if (EMBED) {
    const long long id = p.ids[row];
    erow = static_cast<const T*>(p.table) + size_t(id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id)) * p.ld;
    if (p.freq) pos = float(p.positions[row]);
  }
#pragma unroll
  for (int k = 0; k < U; k++) {
    const int i = threadIdx.x + k * blockDim.x;
    if (!POST) u[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < units) {
      if (EMBED) {
        const float4 e = load4(erow + i * 4);
        float pv[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < 2; j++) {
          const int c = i * 4 + 2 * j;
          if (p.freq && c < p.width) {
            float s, co;
            sincos_turns(pos, p.freq[c / 2], &s, &co);
            pv[2 * j] = s;
            if (c + 1 < p.width) pv[2 * j + 1] = co;
          }
        }
        u[k] = make_float4(fmaf(e.x, p.embed_scale, pv[0]), fmaf(e.y, p.embed_scale, pv[1]), fmaf(e.z, p.embed_scale, pv[2]), fmaf(e.w, p.embed_scale, pv[3]));
        if (p.x0) store4(p.x0 + row * p.ld + i * 4, u[k]);
      } else if (POST) {
        add4(u[k], b[POST ? k : 0]);
      } else {
        u[k] = load4(xr + i * 4);
        float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
        if (p.y1) b = load4(p.y1 + row * p.ld + i * 4);
        if (p.y2) add4(b, load4(p.y2 + row * p.ld + i * 4));
        if (p.routed) {
          const T* ro = static_cast<const T*>(p.routed) + i * 4;
#pragma unroll 4
          for (int j = 0; j < p.top; j++) fma4(b, sw[j], load4(ro + size_t(sp[j]) * p.ld));
        }
        add4(u[k], b);
        if (p.x0) add4(u[k], load4(p.x0 + row * p.ld + i * 4));
      }
      if (p.step) add4(u[k], load4(p.step + i * 4));
      if (!p.last) store4(xr + i * 4, u[k]);
      ss += u[k].x * u[k].x + u[k].y * u[k].y + u[k].z * u[k].z + u[k].w * u[k].w;   // pad columns hold zeros
    }
  }
  float r = 1.0f;
  if (p.g1 || p.g2) {
    warp_part(ss, red);
    __syncthreads();
    r = 1.0f / sqrtf(block_total(red) / float(p.width) + p.eps);
  } else if (p.out_place) {
    __syncthreads();
  }
  if (!p.h1 && !p.h2) return;
  float* shift = nullptr;
  if (p.mu) {
    shift = p.shift + size_t(p.segs[4 * blockIdx.x + 2]) * p.ld;
    fresh = p.positions[row] == 0;
  }
#pragma unroll
  for (int k = 0; k < U; k++) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < units) {
      float4 v = u[k];
      if (p.g1) {
        const float4 g = load4(p.g1 + i * 4);
        v = make_float4(u[k].x * r * g.x, u[k].y * r * g.y, u[k].z * r * g.z, u[k].w * r * g.w);
      }
      if constexpr (NEAR) {
        float4 c = make_float4(0.f, 0.f, 0.f, 0.f), in[kNear], w[kNear];    // loads before stores: one round trip
#pragma unroll
        for (int j = 0; j < kNear; j++)
          if (j < p.taps - 1) {
            w[j] = load4(p.near + size_t(j) * p.ld + i * 4);
            in[j] = kEarly ? pre[kEarly ? k : 0][j] : (fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(past + size_t(j) * p.ld + i * 4));
          }
#pragma unroll
        for (int j = 0; j < kNear; j++)
          if (j < p.taps - 1) {
            mul_add4(c, w[j], in[j]);
            if (j > 0) store4(past + size_t(j - 1) * p.ld + i * 4, in[j]);
          }
        for (int j = kNear; j < p.taps - 1; j++) {
          const float4 x = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(past + size_t(j) * p.ld + i * 4);
          mul_add4(c, load4(p.near + size_t(j) * p.ld + i * 4), x);
          store4(past + size_t(j - 1) * p.ld + i * 4, x);
        }
        mul_add4(c, load4(p.near + size_t(p.taps - 1) * p.ld + i * 4), v);
        if (p.taps > 1) store4(past + size_t(p.taps - 2) * p.ld + i * 4, v);
        add4(v, c);
      }
      const size_t off = size_t(blockIdx.x) * p.ldh + i * 4;
      if (p.mu) {
        const float4 prev = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(shift + i * 4);
        store4(shift + i * 4, v);
        for (int s = 0; s < p.nmix; s++)
          store4(static_cast<T*>(p.mixes) + (row * p.nmix + s) * p.ld + i * 4, mix4(v, prev, load4(p.mu + size_t(s) * p.ld + i * 4)));
      } else if (!p.h1) {
      } else if (p.out_place) {
        for (int j = 0; j < p.out_top; j++) store4(static_cast<T*>(p.h1) + size_t(so[j]) * p.ldh + i * 4, v);
      } else if (p.h1_f32) {
        store4(static_cast<float*>(p.h1) + off, v);
      } else {
        store4(static_cast<T*>(p.h1) + off, v);
      }
      if (p.g2) {
        const float4 g2 = load4(p.g2 + i * 4);
        store4(static_cast<T*>(p.h2) + off, make_float4(u[k].x * r * g2.x, u[k].y * r * g2.y, u[k].z * r * g2.z, u[k].w * r * g2.w));
      }
    }
  }
}

// mixes[t][s] = h_t + (h_{t-1} - h_t) * mu_s; the row before a segment's first comes from the state (zeros at a sequence's start).  The state is
// read only: the recurrence of the layer, which runs later, replaces it.
template <typename T>
__global__ void __launch_bounds__(256) k_token_shift(const float* __restrict__ h, const float* __restrict__ mu, const float* __restrict__ shift,
                                                     T* __restrict__ mixes, const int* __restrict__ segs, const int* __restrict__ seg_of_row,
                                                     const int* __restrict__ positions, int ld, int nmix) {
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int row = blockIdx.x, i = (blockIdx.y * 256 + threadIdx.x) * 4;
  if (i >= ld) return;
  const int* sg = segs + 4 * (seg_of_row ? seg_of_row[row] : row);
  const float4 v = load4(h + size_t(row) * ld + i);
  float4 prev = make_float4(0.f, 0.f, 0.f, 0.f);
  if (row > sg[0]) prev = load4(h + size_t(row - 1) * ld + i);
  else if (positions[row] != 0) prev = load4(shift + size_t(sg[2]) * ld + i);
  for (int s = 0; s < nmix; s++) store4(mixes + (size_t(row) * nmix + s) * ld + i, mix4(v, prev, load4(mu + size_t(s) * ld + i)));
}

template <typename T, bool EMBED, bool POST, bool NEAR>
cudaError_t launch_n(const ResidualParams& p, int rows, cudaStream_t st) {
  const int units = p.ld / 4;
  const int per = units <= 64 ? 1 : (units <= kThreads * 2 ? 2 : (units <= kThreads * 4 ? 4 : (units <= kThreads * 8 ? 8 : 16)));
  int threads = ((units + per - 1) / per + 31) / 32 * 32;
  if (threads > kThreads) return cudaErrorInvalidValue;
  if (threads < kMaxTop) threads = kMaxTop;
  const dim3 grid(rows), blk(threads);
  switch (per) {
    case 1: return pdl::launch(k_residual<T, EMBED, POST, NEAR, 1>, grid, blk, 0, st, 1, p);
    case 2: return pdl::launch(k_residual<T, EMBED, POST, NEAR, 2>, grid, blk, 0, st, 1, p);
    case 4: return pdl::launch(k_residual<T, EMBED, POST, NEAR, 4>, grid, blk, 0, st, 1, p);
    case 8: return pdl::launch(k_residual<T, EMBED, POST, NEAR, 8>, grid, blk, 0, st, 1, p);
    default: return pdl::launch(k_residual<T, EMBED, POST, NEAR, 16>, grid, blk, 0, st, 1, p);
  }
}
template <typename T, bool EMBED, bool POST>
cudaError_t launch_u(const ResidualParams& p, int rows, cudaStream_t st) {
  return p.near ? launch_n<T, EMBED, POST, true>(p, rows, st) : launch_n<T, EMBED, POST, false>(p, rows, st);
}
template <typename T>
cudaError_t launch_t(const ResidualParams& p, int rows, cudaStream_t st) {
  if (p.ids) return launch_u<T, true, false>(p, rows, st);
  return p.post ? launch_u<T, false, true>(p, rows, st) : launch_u<T, false, false>(p, rows, st);
}

}  // namespace

extern "C" {

// See the top of the file.  ids != null: the embedding (y1, y2, routed ignored; freq null: no position vector).  mu != null: the mixes are written
// instead of h1.  post != null: the branches' norm (y2, x0, step and mixes do not go with it).  weight null: every weight is weight_const.  g1 null: h1 = x;
// h1 null: not written.  near != null: the convolution of one row per segment is added to h1.
int tbv_op_residual(const void* ids, const void* table, const void* freq, const void* positions, float embed_scale, long long vocab, void* x,
                    void* x0, const void* y1, const void* y2, const void* step, const void* routed, const void* place, const void* weight, int top,
                    const void* g1, const void* g2, void* h1, void* h2, int h1_f32, const void* row_map, int last, const void* mu, void* mixes,
                    void* shift, const void* segs, int nmix, const void* post, const void* sums, int nsum, int sum_width, float weight_const, const void* out_place,
                    int out_top, const void* near, void* past, int taps, int rows, int width, int ld, int ldh, float eps, int bf16, void* stream) {
  if (rows <= 0) return 0;
  if (width <= 0 || width > ld || (ld % 4) || (ldh % 4) || ld > kThreads * 4 * kMaxUnits || ldh < ld || (routed && (top < 1 || top > kMaxTop))) return -2;
  if (post && (ids || y2 || x0 || step || mu)) return -2;
  if ((sums && (!post || nsum <= 0 || sum_width <= 0)) || (out_place && (last || (h1_f32 && bf16) || mu || out_top < 1 || out_top > kMaxTop))) return -2;
  if (!h1 && (last || out_place || near)) return -2;
  if (near && (last || mu || !segs || !positions || taps < 1 || (taps > 1 && !past))) return -2;
  if (mu && (!g1 || last || !segs || !positions || !shift || !mixes)) return -2;
  ResidualParams p{};
  p.ids = static_cast<const long long*>(ids); p.table = table; p.freq = static_cast<const float2*>(freq); p.positions = static_cast<const int*>(positions);
  p.embed_scale = embed_scale; p.vocab = vocab;
  p.x = static_cast<float*>(x); p.x0 = static_cast<float*>(x0); p.y1 = static_cast<const float*>(y1); p.y2 = static_cast<const float*>(y2);
  p.step = static_cast<const float*>(step); p.routed = routed; p.place = static_cast<const int*>(place); p.weight = static_cast<const float*>(weight); p.weight_const = weight_const; p.top = top;
  p.post = static_cast<const float*>(post); p.sums = static_cast<const float*>(sums); p.nsum = nsum; p.sum_width = sum_width;
  p.out_place = static_cast<const int*>(out_place); p.out_top = out_top;
  p.g1 = static_cast<const float*>(g1); p.g2 = static_cast<const float*>(g2); p.h1 = h1; p.h2 = h2; p.h1_f32 = h1_f32;
  p.rows = static_cast<const long long*>(row_map); p.last = last; p.mu = static_cast<const float*>(mu); p.mixes = mixes; p.shift = static_cast<float*>(shift);
  p.near = static_cast<const float*>(near); p.past = static_cast<float*>(past); p.taps = taps;
  p.segs = static_cast<const int*>(segs); p.nmix = nmix; p.width = width; p.ld = ld; p.ldh = ldh; p.eps = eps;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = bf16 ? launch_t<__nv_bfloat16>(p, rows, st) : launch_t<float>(p, rows, st);
  return e == cudaSuccess ? 0 : -1;
}

// h fp32 [rows, ld] -> mixes [rows, nmix, ld]
int tbv_op_token_shift(const void* h, const void* mu, const void* shift, void* mixes, const void* segs, const void* seg_of_row, const void* positions,
                       int rows, int ld, int nmix, int bf16, void* stream) {
  if (rows <= 0) return 0;
  if (ld % 4) return -2;
  const dim3 grid(rows, (ld / 4 + 255) / 256);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const float *hf = static_cast<const float*>(h), *m = static_cast<const float*>(mu), *s = static_cast<const float*>(shift);
  const int *sg = static_cast<const int*>(segs), *so = static_cast<const int*>(seg_of_row), *po = static_cast<const int*>(positions);
  cudaError_t e = bf16 ? pdl::launch(k_token_shift<__nv_bfloat16>, grid, dim3(256), 0, st, 1, hf, m, s, static_cast<__nv_bfloat16*>(mixes), sg, so, po, ld, nmix)
                       : pdl::launch(k_token_shift<float>, grid, dim3(256), 0, st, 1, hf, m, s, static_cast<float*>(mixes), sg, so, po, ld, nmix);
  return e == cudaSuccess ? 0 : -1;
}

}  // extern "C"
