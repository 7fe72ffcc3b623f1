// hyper.cu — residual streams with hyper-connections, fused with the layer scale before and the RMSNorm after.
//
// A model may carry S residual streams x_1..x_S (fp32) instead of one.  A sublayer reads u = sum_s in[s] x_s, and its
// result y goes back as  x_t <- sum_s mix[s][t] x_s + out[t] * (scale * y)  for all t at once (mix is indexed [from][to]).  One
// kernel does the write-back of a sublayer AND the read + norm of the next, so the streams cross HBM once per sublayer:
//
//   k_hyper<kEmbed>  x_s = embed[id] * scale for every s;            h = norm(sum_s in[s] x_s) * gamma
//   k_hyper<kMix>    x_t = sum_s mix[s][t] x_s + out[t] * ls * y;     h = norm(sum_t in[t] x_t) * gamma
//   k_hyper<kLast>   as kMix for selected rows, the streams not stored (in = 1 gives the plain sum)
//
// S = 1 with in = mix = out = 1 is the ordinary residual stream.  All arithmetic is fp32; h is stored as bf16 or fp32.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../pdl.cuh"

namespace {

constexpr int kMaxStreams = 8;
constexpr int kThreads = 512;
constexpr int kMaxUnits = 16;     // float4 units of a row per thread: width <= 512 * 16 * 4
enum Mode : int { kEmbed = 0, kMix = 1, kLast = 2 };

struct HyperParams {
  const long long* ids;     // kEmbed: token ids
  const void* table;        // kEmbed: [vocab, ld] in the activation type
  float embed_scale;
  long long vocab;
  float* x;                 // [rows, S, ld]
  const float* y;           // [rows, ld] sublayer result
  const float* ls;          // [ld] layer scale
  const float *hout, *hmix; // [S], [S * S] of the sublayer that ends
  const float* hin;         // [S] of the sublayer that follows
  const float* gamma;       // [ld] norm weight that follows
  const long long* rows;    // kLast: source row of every output row (null = identity)
  void* h;                  // [rows, ldh]
  int width, ld, ldh, bf16;
  float eps;
};

__device__ __forceinline__ float4 load_emb(const void* t, size_t off, int bf16) {
  if (!bf16) return *reinterpret_cast<const float4*>(static_cast<const float*>(t) + off);
  const uint2 v = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(t) + off);
  return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void fma4(float4& a, float s, const float4& b) {
  a.x = fmaf(s, b.x, a.x); a.y = fmaf(s, b.y, a.y); a.z = fmaf(s, b.z, a.z); a.w = fmaf(s, b.w, a.w);
}

template <int MODE, int S, int U>
__global__ void __launch_bounds__(kThreads) k_hyper(const HyperParams p) {
  __shared__ float red[32];
  __shared__ float coef[kMaxStreams * kMaxStreams + 2 * kMaxStreams];
  pdl::launch_dependents();
  // the coefficients are weights: no need to wait for the kernel before
  if (threadIdx.x < S) {
    coef[threadIdx.x] = p.hin[threadIdx.x];
    if (MODE != kEmbed) coef[S + threadIdx.x] = p.hout[threadIdx.x];
  }
  if (MODE != kEmbed && threadIdx.x < S * S) coef[2 * S + threadIdx.x] = p.hmix[threadIdx.x];
  pdl::grid_dependency_wait();
  __syncthreads();
  const int units = p.ld / 4;
  const size_t row = MODE == kLast && p.rows ? size_t(p.rows[blockIdx.x]) : blockIdx.x;
  float* xr = p.x + row * S * p.ld;
  float4 u[U];
  float ss = 0.f;
  size_t erow = 0;
  if (MODE == kEmbed) {
    const long long id = p.ids[row];
    erow = size_t(id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id)) * p.ld;
  }
#pragma unroll
  for (int k = 0; k < U; k++) {
    const int i = threadIdx.x + k * blockDim.x;
    u[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < units) {
      if (MODE == kEmbed) {
        float4 e = load_emb(p.table, erow + i * 4, p.bf16);
        e.x *= p.embed_scale; e.y *= p.embed_scale; e.z *= p.embed_scale; e.w *= p.embed_scale;
#pragma unroll
        for (int s = 0; s < S; s++) {
          *reinterpret_cast<float4*>(xr + size_t(s) * p.ld + i * 4) = e;
          fma4(u[k], coef[s], e);
        }
      } else {
        float4 xs[S], y = *reinterpret_cast<const float4*>(p.y + row * p.ld + i * 4);
        const float4 l = *reinterpret_cast<const float4*>(p.ls + i * 4);
        y.x *= l.x; y.y *= l.y; y.z *= l.z; y.w *= l.w;
#pragma unroll
        for (int s = 0; s < S; s++) xs[s] = *reinterpret_cast<const float4*>(xr + size_t(s) * p.ld + i * 4);
#pragma unroll
        for (int t = 0; t < S; t++) {
          float4 n = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int s = 0; s < S; s++) fma4(n, coef[2 * S + s * S + t], xs[s]);
          fma4(n, coef[S + t], y);
          if (MODE == kMix) *reinterpret_cast<float4*>(xr + size_t(t) * p.ld + i * 4) = n;
          fma4(u[k], coef[t], n);
        }
      }
      ss += u[k].x * u[k].x + u[k].y * u[k].y + u[k].z * u[k].z + u[k].w * u[k].w;   // pad columns hold zeros
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int w = 0; w < int(blockDim.x + 31) / 32; w++) tot += red[w];
  const float r = 1.0f / sqrtf(tot / float(p.width) + p.eps);
#pragma unroll
  for (int k = 0; k < U; k++) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < units) {
      const float4 g = *reinterpret_cast<const float4*>(p.gamma + i * 4);
      const float4 v = make_float4(u[k].x * r * g.x, u[k].y * r * g.y, u[k].z * r * g.z, u[k].w * r * g.w);
      const size_t off = size_t(blockIdx.x) * p.ldh + i * 4;
      if (p.bf16) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        uint2 pk;
        pk.x = *reinterpret_cast<uint32_t*>(&lo);
        pk.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p.h) + off) = pk;
      } else {
        *reinterpret_cast<float4*>(static_cast<float*>(p.h) + off) = v;
      }
    }
  }
}

template <int MODE, int S>
cudaError_t launch_u(const HyperParams& p, int rows, cudaStream_t st) {
  const int units = p.ld / 4;
  // two units per thread while the row allows it: enough loads in flight without a second wave of CTAs
  const int per = units <= 64 ? 1 : (units <= kThreads * 2 ? 2 : (units <= kThreads * 4 ? 4 : (units <= kThreads * 8 ? 8 : 16)));
  const int threads = ((units + per - 1) / per + 31) / 32 * 32;
  if (threads > kThreads) return cudaErrorInvalidValue;
  const dim3 grid(rows), blk(threads);
  switch (per) {
    case 1: return pdl::launch(k_hyper<MODE, S, 1>, grid, blk, 0, st, 1, p);
    case 2: return pdl::launch(k_hyper<MODE, S, 2>, grid, blk, 0, st, 1, p);
    case 4: return pdl::launch(k_hyper<MODE, S, 4>, grid, blk, 0, st, 1, p);
    case 8: return pdl::launch(k_hyper<MODE, S, 8>, grid, blk, 0, st, 1, p);
    default: return pdl::launch(k_hyper<MODE, S, 16>, grid, blk, 0, st, 1, p);
  }
}
template <int MODE>
int launch_s(const HyperParams& p, int rows, int streams, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (p.width <= 0 || p.width > p.ld || (p.ld % 4) || (p.ldh % 4) || p.ld > kThreads * 4 * kMaxUnits || p.ldh < p.ld) return -2;
  cudaError_t e;
  switch (streams) {
    case 1: e = launch_u<MODE, 1>(p, rows, st); break;
    case 2: e = launch_u<MODE, 2>(p, rows, st); break;
    case 3: e = launch_u<MODE, 3>(p, rows, st); break;
    case 4: e = launch_u<MODE, 4>(p, rows, st); break;
    case 5: e = launch_u<MODE, 5>(p, rows, st); break;
    case 6: e = launch_u<MODE, 6>(p, rows, st); break;
    case 7: e = launch_u<MODE, 7>(p, rows, st); break;
    case 8: e = launch_u<MODE, 8>(p, rows, st); break;
    default: return -2;
  }
  return e == cudaSuccess ? 0 : -1;
}

}  // namespace

extern "C" {

// x: fp32 [rows, streams, ld]; every stream of row r := table[ids[r]] * scale; h := norm(sum_s hin[s] x_s) * gamma.
int tbv_op_hyper_embed(const void* ids, const void* table, long long vocab, float scale, void* x, const void* hin, const void* gamma,
                       void* h, int rows, int streams, int width, int ld, int ldh, float eps, int bf16, void* stream) {
  HyperParams p{};
  p.ids = static_cast<const long long*>(ids); p.table = table; p.vocab = vocab; p.embed_scale = scale;
  p.x = static_cast<float*>(x); p.hin = static_cast<const float*>(hin); p.gamma = static_cast<const float*>(gamma);
  p.h = h; p.width = width; p.ld = ld; p.ldh = ldh; p.eps = eps; p.bf16 = bf16;
  return launch_s<kEmbed>(p, rows, streams, static_cast<cudaStream_t>(stream));
}

// Ends one sublayer (y: its result, fp32 [rows, ld]) and starts the next.  last != 0: rows[r] selects the source row of output
// row r (null = identity) and the streams are left as they are.
int tbv_op_hyper_mix(const void* y, const void* ls, const void* hout, const void* hmix, void* x, const void* hin, const void* gamma,
                     void* h, const void* row_map, int last, int rows, int streams, int width, int ld, int ldh, float eps, int bf16,
                     void* stream) {
  HyperParams p{};
  p.y = static_cast<const float*>(y); p.ls = static_cast<const float*>(ls); p.hout = static_cast<const float*>(hout);
  p.hmix = static_cast<const float*>(hmix); p.x = static_cast<float*>(x); p.hin = static_cast<const float*>(hin);
  p.gamma = static_cast<const float*>(gamma); p.h = h; p.rows = static_cast<const long long*>(row_map);
  p.width = width; p.ld = ld; p.ldh = ldh; p.eps = eps; p.bf16 = bf16;
  return last ? launch_s<kLast>(p, rows, streams, static_cast<cudaStream_t>(stream))
              : launch_s<kMix>(p, rows, streams, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
