// shared_attn.cu — grouped-query attention whose values are the keys before their norm, with a query temperature that grows with the position
// and soft-capped scores.
//
// A key is its value times one factor (the reciprocal root mean square over the head) times a weight per channel.  The weight and the
// score scale are folded into the query, so ONE cached row per token and key head serves as key and as value:
//   row = dim values | fp32 factor | pad          (dim padded to 16; eight places behind it, as in the latent cache)
//   score(i, j) = cap * tanh((q'_i . row_j) * factor_j / cap),  q' = norm(q) * temperature * fold
// Rows of a block lie together per key head ([blocks, kv_heads, block_size, dim + 8]), so that the rows form (latent_attn.cu, template KS)
// brings a block in with one bulk copy.  Here: the kernel that normalises queries and writes cache rows, the prefill form, and a rows form for heads
// of up to 128 channels in which every warp walks blocks of its own: a row is small, so that the barriers of a CTA-wide tile would cost
// more than its work.
//
// The same kernels (template PAIR) serve attention whose cached row holds a key and a value of sizes of their own,
//   row = Dp key channels | Vp value channels | pad
// with queries and keys normed over all heads of the projection at once, a rotation of the first dimensions (interleaved pairs) or none, optionally
// soft-capped scores, a sliding window or chunks of positions (keys before the first visible one are not read), and a sigmoid gate on the result.
// A second kernel writes such rows with norms per head and values mixed with those of another layer (k_head_prep).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>

#include "../pdl.cuh"
#include "attn_mma.cuh"
#include "ops.h"
#include "sm100.cuh"
#include "vec.cuh"

using namespace attn_mma;
using vec::from_f;
using vec::to_f;

namespace {

constexpr int kRowPad = 8;

struct PrepParams {
  void* qk;                 // [rows, ldq]: heads * Dp query columns, kv_heads * Dp key columns
  void* qa;                 // [n_rows_form, heads, Dp + pad]; the queries of later rows stay in place
  void* cache;
  const float* fold;        // [Dp]
  const int* positions;
  const long long* slots;
  int rows, ldq, heads, kv_heads, dim, Dp, n_rows_form, block_size;
  float eps, temp_coef;
  double temp_every;
};

// one warp per (row, head); heads of keys come after those of queries
template <typename T>
__global__ void __launch_bounds__(256) k_shared_prep(const PrepParams p) {
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int lane = threadIdx.x & 31, nh = p.heads + p.kv_heads;
  const long long w = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (w >= (long long)p.rows * nh) return;
  const int row = int(w / nh), h = int(w - (long long)row * nh);
  T* src = static_cast<T*>(p.qk) + size_t(row) * p.ldq + size_t(h) * p.Dp;
  float ss = 0.f;
  for (int i = lane; i < p.dim; i += 32) { const float v = to_f(src[i]); ss = fmaf(v, v, ss); }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float r = 1.0f / sqrtf(ss / float(p.dim) + p.eps);
  if (h < p.heads) {
    const double turns = floor((double(p.positions[row]) + 1.0) / p.temp_every);
    const float f = r * (1.0f + p.temp_coef * logf(float(turns) + 1.0f));
    T* dst = row < p.n_rows_form ? static_cast<T*>(p.qa) + (size_t(row) * p.heads + h) * (p.Dp + kRowPad) : src;
    for (int i = lane; i < p.Dp; i += 32) from_f(dst[i], to_f(src[i]) * f * p.fold[i]);
  } else {
    const long long slot = p.slots[row];
    if (slot < 0) return;
    const size_t at = size_t((slot / p.block_size * p.kv_heads + (h - p.heads)) * p.block_size + slot % p.block_size);
    T* dst = static_cast<T*>(p.cache) + at * (p.Dp + kRowPad);
    for (int i = lane; i < p.Dp; i += 32) dst[i] = src[i];
    if (lane == 0) *reinterpret_cast<float*>(dst + p.Dp) = r;
  }
}

// Paired rows.  One CTA per token: square sums over all query and all key columns, then norm, rotation and the writes.
constexpr int kMaxPairs = 512;
struct PairPrepParams {
  void* wide;               // [rows, ldw]: heads * Dp query columns, kv_heads * Dp key columns, kv_heads * Vp value columns
  void* qa;                 // [n_rows_form, heads, Dp + pad]; the queries of later rows stay in place
  void* cache;
  const float *qn, *kn;     // [heads * Dp], [kv_heads * Dp]
  const float2* turns;      // [pairs]: turns per position, high and low part
  const int* positions;
  const long long* slots;
  int ldw, heads, kv_heads, dim, Dp, Vp, pairs, n_rows_form, block_size;
  float eps;
};
template <typename T>
__global__ void __launch_bounds__(256) k_paired_prep(const PairPrepParams p) {
  __shared__ float cs[kMaxPairs], sn[kMaxPairs], red[2][8];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int row = blockIdx.x, tid = threadIdx.x, K = p.heads * p.Dp, G = p.kv_heads;
  T* q = static_cast<T*>(p.wide) + size_t(row) * p.ldw;
  const T* k = q + K;
  if (p.pairs) {
    const float pos = float(p.positions[row]);
    for (int i = tid; i < p.pairs; i += 256) vec::sincos_turns(pos, p.turns[i], &sn[i], &cs[i]);
  }
  float sq = 0.f, sk = 0.f;                     // pad channels hold zeros
  for (int i = tid * 8; i < K; i += 2048) {
    float f[8];
    vec::load8(q + i, f);
#pragma unroll
    for (int e = 0; e < 8; e++) sq = fmaf(f[e], f[e], sq);
  }
  for (int i = tid * 8; i < G * p.Dp; i += 2048) {
    float f[8];
    vec::load8(k + i, f);
#pragma unroll
    for (int e = 0; e < 8; e++) sk = fmaf(f[e], f[e], sk);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sk += __shfl_xor_sync(0xffffffffu, sk, o);
  }
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) { sq += red[0][w]; sk += red[1][w]; }
  const float rq = 1.0f / sqrtf(sq / float(p.heads * p.dim) + p.eps);
  auto finish = [&](float* f, float r, const float* weight, int d) {     // eight channels from channel d of a head
    float w[8];
    vec::load8(weight, w);
#pragma unroll
    for (int e = 0; e < 8; e++) f[e] *= r * w[e];
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      const int i = (d + e) / 2;
      if (i < p.pairs) {
        const float u = f[e], v = f[e + 1], c = cs[i], s = sn[i];
        f[e] = u * c - v * s;
        f[e + 1] = v * c + u * s;
      }
    }
  };
  for (int i = tid * 8; i < K; i += 2048) {
    const int h = i / p.Dp, d = i - h * p.Dp;
    float f[8];
    vec::load8(q + i, f);
    finish(f, rq, p.qn + i, d);
    vec::store8(row < p.n_rows_form ? static_cast<T*>(p.qa) + (size_t(row) * p.heads + h) * (p.Dp + kRowPad) + d : q + i, f);
  }
  const long long slot = G ? p.slots[row] : -1;
  if (slot < 0) return;
  const float rk = 1.0f / sqrtf(sk / float(G * p.dim) + p.eps);
  const int len = p.Dp + p.Vp + kRowPad;
  auto dst = [&](int g) { return static_cast<T*>(p.cache) + size_t((slot / p.block_size * G + g) * p.block_size + slot % p.block_size) * len; };
  for (int i = tid * 8; i < G * p.Dp; i += 2048) {
    const int g = i / p.Dp, d = i - g * p.Dp;
    float f[8];
    vec::load8(k + i, f);
    finish(f, rk, p.kn + i, d);
    vec::store8(dst(g) + d, f);
  }
  const T* v = k + G * p.Dp;
  for (int i = tid * 8; i < G * p.Vp; i += 2048) {
    const int g = i / p.Vp;
    vec::Raw8<T> f;
    f.load(v + i);
    f.store(dst(g) + p.Dp + i - g * p.Vp);
  }
}

// Paired rows with norms per head and without weights, a factor per query head, and values that may be mixed with those of another layer:
//   v <- (1 - lambda) v + lambda v_first        v_first: what the first of these layers stored for the same token
// Groups of lanes share a head, 8 channels per lane: heads of queries, keys and values one after the other.
struct HeadPrepParams {
  void* wide;               // [rows, ldw]: heads * Dp query columns, kv_heads * Dp key columns, kv_heads * Vp value columns
  void* qa;                 // as above
  void* cache;
  const float* qscale;      // [heads]
  const float2* turns;      // [pairs]
  const int* positions;
  const long long* slots;
  void* v_first;            // [rows, kv_heads * Vp] or null
  const float* lambda;      // null: this layer's values are stored in v_first
  int rows, ldw, heads, kv_heads, dim, Dp, Vp, pairs, n_rows_form, block_size;
  float eps;
};
template <typename T, int GS>             // lanes per head
__global__ void __launch_bounds__(256) k_head_prep(const HeadPrepParams p) {
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int l = threadIdx.x % GS, H = p.heads, G = p.kv_heads, nh = H + 2 * G;
  const long long item = (long long)blockIdx.x * (256 / GS) + threadIdx.x / GS;
  const bool on = item < (long long)p.rows * nh;                    // all lanes take part in the exchanges
  const int row = on ? int(item / nh) : 0, h = on ? int(item - (long long)row * nh) : 0;
  T* src = static_cast<T*>(p.wide) + size_t(row) * p.ldw;
  const long long slot = p.slots[row];
  auto cached = [&](int g) {
    return static_cast<T*>(p.cache) + size_t((slot / p.block_size * G + g) * p.block_size + slot % p.block_size) * (p.Dp + p.Vp + kRowPad);
  };
  float ss = 0.f;
  if (on && h < H + G) {
    src += size_t(h) * p.Dp;
    for (int i = l * 8; i < p.Dp; i += GS * 8) {
      float f[8];
      vec::load8(src + i, f);
#pragma unroll
      for (int e = 0; e < 8; e++) ss = fmaf(f[e], f[e], ss);        // pad channels hold zeros
    }
  }
#pragma unroll
  for (int o = GS / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!on) return;
  if (h < H + G) {
    float r = 1.0f / sqrtf(ss / float(p.dim) + p.eps);
    if (h < H) r *= p.qscale[h];
    else if (slot < 0) return;
    T* dst = h < H ? (row < p.n_rows_form ? static_cast<T*>(p.qa) + (size_t(row) * H + h) * (p.Dp + kRowPad) : src) : cached(h - H);
    const float pos = float(p.positions[row]);
    for (int i = l * 8; i < p.Dp; i += GS * 8) {
      float f[8];
      vec::load8(src + i, f);
#pragma unroll
      for (int e = 0; e < 8; e += 2) {
        float u = f[e] * r, v = f[e + 1] * r;
        if ((i + e) / 2 < p.pairs) {
          float sn, cs;
          vec::sincos_turns(pos, p.turns[(i + e) / 2], &sn, &cs);
          const float a = u * cs - v * sn;
          v = v * cs + u * sn;
          u = a;
        }
        f[e] = u;
        f[e + 1] = v;
      }
      vec::store8(dst + i, f);
    }
    return;
  }
  const int g = h - H - G;
  src += size_t(H + G) * p.Dp + size_t(g) * p.Vp;
  T* first = p.v_first ? static_cast<T*>(p.v_first) + (size_t(row) * G + g) * p.Vp : nullptr;
  const float lam = p.v_first && p.lambda ? *p.lambda : 0.f;
  for (int i = l * 8; i < p.Vp; i += GS * 8) {
    float f[8];
    vec::load8(src + i, f);
    if (first && p.lambda) {
      float a[8];
      vec::load8(first + i, a);
#pragma unroll
      for (int e = 0; e < 8; e++) f[e] = fmaf(lam, a[e], (1.0f - lam) * f[e]);
    } else if (first) {
      vec::store8(first + i, f);
    }
    if (slot >= 0) vec::store8(cached(g) + p.Dp + i, f);
  }
}
template <typename T>
cudaError_t launch_head_prep(const HeadPrepParams& p, cudaStream_t st) {
  const int units = (p.Dp > p.Vp ? p.Dp : p.Vp) / 8;
  const long long items = (long long)p.rows * (p.heads + 2 * p.kv_heads);
  auto grid = [&](int gs) { return dim3(unsigned((items + 256 / gs - 1) / (256 / gs))); };
  if (units <= 4) return pdl::launch(k_head_prep<T, 4>, grid(4), dim3(256), 0, st, 1, p);
  if (units <= 8) return pdl::launch(k_head_prep<T, 8>, grid(8), dim3(256), 0, st, 1, p);
  if (units <= 16) return pdl::launch(k_head_prep<T, 16>, grid(16), dim3(256), 0, st, 1, p);
  return pdl::launch(k_head_prep<T, 32>, grid(32), dim3(256), 0, st, 1, p);
}

// ---- rows form ---------------------------------------------------------------------------------------------------------
struct RowsParams {
  const __nv_bfloat16 *qa, *cache;
  __nv_bfloat16* out;       // [rows, heads, Vp]
  const int *tables, *seq_of_row, *ctx_lens;
  int heads, kv_heads, Dp, Vp, block_size, max_blocks, splits;   // Vp = Dp where one row serves as key and value
  float softcap;
  int* err;
  int window, chunk;        // attn_mma::first_visible (PAIR)
  const __nv_bfloat16* gate;   // [rows, ldg]: column h * Vp (PAIR; null: none)
  int ldg;
};
__device__ __forceinline__ float4 gated(float4 a, const __nv_bfloat16* gate) {
  const float4 g = load_bf16x4(gate);
  return make_float4(a.x * vec::sigmoid<__nv_bfloat16>(g.x), a.y * vec::sigmoid<__nv_bfloat16>(g.y), a.z * vec::sigmoid<__nv_bfloat16>(g.z), a.w * vec::sigmoid<__nv_bfloat16>(g.w));
}

// One row and up to 16 query heads of a key head per CTA; grid (rows, head tiles, splits), cluster (1, 1, splits).  Warp w takes the kTok-token
// units w, w + kWarps, .. of the CTA's token range through a ring of its own, filled by bulk copies of 16 tokens, with a running maximum of its own;
// the warps' results are merged at the end, then those of the cluster, in fixed order.  Tokens (scores) and channels (sums) sit on the M side of the
// products and heads on the N side, eight at a time (NH times): four query heads per key head leave half of the columns idle, not three quarters.
constexpr int kWarps = 4, kStages = 3, kMaxSplits = 8;
template <int NK, int NH, int kTok, bool PAIR>   // steps of 16 channels (keys' and values', at most), tiles of 8 heads
__global__ void __launch_bounds__(kWarps * 32, 2) k_shared_rows(const RowsParams p) {
  extern __shared__ __align__(128) uint8_t dsm[];
  __shared__ unsigned long long full[kWarps][kStages];
  __shared__ float sh_m[kWarps][16], sh_l[kWarps][16], sh_ml[16][2], sh_fac[kMaxSplits][16], sh_sm[kMaxSplits][16];
  __shared__ int abort_flag;
  pdl::launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r8 = lane >> 2, quad = lane & 3;
  if (lane == 0) {
    for (int s = 0; s < kStages; s++) sm100::mbar_init(smem_addr(&full[warp][s]), 1);
    if (warp == 0) abort_flag = 0;
    sm100::mbar_fence_init();
  }
  __syncthreads();
  pdl::grid_dependency_wait();
  const int row = blockIdx.x, sp = blockIdx.z, S = p.splits;
  const int G = p.kv_heads, hpk = p.heads / G, tpg = (hpk + 15) / 16, g = blockIdx.y / tpg;
  const int h0 = g * hpk + (blockIdx.y - g * tpg) * 16, nq = min(16, (g + 1) * hpk - h0);
  const int Vp = PAIR ? p.Vp : p.Dp, voff = PAIR ? p.Dp : 0, ksteps = p.Dp / 16, vsteps = Vp / 16;
  const int qlen = p.Dp + kRowPad, rowlen = qlen + (PAIR ? Vp : 0), pitch = rowlen * 2;
  const int ctx = min(p.ctx_lens[row], p.max_blocks * p.block_size);
  const int* bt = p.tables + size_t(p.seq_of_row ? p.seq_of_row[row] : row) * p.max_blocks;
  const int lo = PAIR ? first_visible(ctx, p.window, p.chunk) : 0, from = lo & ~15;
  int chunk = (ctx - from + S - 1) / S;
  chunk = (chunk + kTok - 1) / kTok * kTok;
  const int t0 = min(ctx, from + sp * chunk), t1 = min(ctx, t0 + chunk);
  const int units = (t1 - t0 + kTok - 1) / kTok, mine = units > warp ? (units - warp + kWarps - 1) / kWarps : 0;

  // blocks of this warp's unit i: looked up for kAhead units at a time, a lane per 16 tokens
  constexpr int kPieces = kTok / 16, kAhead = 32 / kPieces;
  int entry = 0;
  auto look_up = [&](int i0) {
    const int tok = t0 + (warp + kWarps * (i0 + lane / kPieces)) * kTok + lane % kPieces * 16;
    return tok < t1 ? bt[tok / p.block_size] : 0;
  };
  const uint32_t ring = smem_addr(dsm) + uint32_t(warp) * kStages * kTok * pitch;
  auto issue = [&](int i) {               // whole warp; unit i of this warp into its stage
    if (i >= mine) return;
    if (i % kAhead == 0) entry = look_up(i);
    const int block = __shfl_sync(0xffffffffu, entry, i % kAhead * kPieces + lane % kPieces);
    const int tok = t0 + (warp + kWarps * i) * kTok, n = min(kTok, t1 - tok);
    const uint32_t bar = smem_addr(&full[warp][i % kStages]);
    if (lane == 0) sm100::mbar_expect_tx(bar, uint32_t(n) * pitch);
    __syncwarp();
    if (lane * 16 < n) {                   // lanes 0 .. kPieces - 1
      const int tk = tok + lane * 16;
      sm100::bulk_load(ring + ((i % kStages) * kTok + lane * 16) * pitch, p.cache + ((size_t(block) * G + g) * p.block_size + tk % p.block_size) * rowlen,
                       uint32_t(min(16, n - lane * 16)) * pitch, bar);
    }
  };
#pragma unroll
  for (int i = 0; i < kStages; i++) issue(i);

  // right operand of the scores: q^T, channels x heads
  uint32_t qf[NK][NH][2];
  const __nv_bfloat16* qa = p.qa + (size_t(row) * p.heads + h0) * qlen + quad * 2;
#pragma unroll
  for (int k = 0; k < NK; k++)
#pragma unroll
    for (int t = 0; t < NH; t++)
#pragma unroll
      for (int j = 0; j < 2; j++)
        qf[k][t][j] = k < ksteps && t * 8 + r8 < nq ? *reinterpret_cast<const uint32_t*>(qa + size_t(t * 8 + r8) * qlen + k * 16 + j * 8) : 0u;
  float o[NK][NH][4];         // channels 16 k + r8 (+ 8), heads 8 t + 2 quad (+ 1)
#pragma unroll
  for (int k = 0; k < NK; k++)
#pragma unroll
    for (int t = 0; t < NH; t++) o[k][t][0] = o[k][t][1] = o[k][t][2] = o[k][t][3] = 0.f;
  float m[NH][2], l[NH][2];
#pragma unroll
  for (int t = 0; t < NH; t++) { m[t][0] = m[t][1] = kNegBig; l[t][0] = l[t][1] = 0.f; }

  int done = 0;
  for (; done < mine; done++) {
    const int i = done, n = min(kTok, t1 - t0 - (warp + kWarps * i) * kTok);
    const uint32_t sk = ring + (i % kStages) * kTok * pitch;
    if (!__all_sync(0xffffffffu, sm100::mbar_wait(smem_addr(&full[warp][i % kStages]), uint32_t(i / kStages) & 1u, &abort_flag, 2000000000ull))) break;
    if (n < kTok) {                        // missing rows: a weight of zero must not meet a stale bit pattern
      for (int r = n; r < kTok; r++)
        for (int c = lane; c < rowlen / 8; c += 32) st_zero16(sk + r * pitch + c * 16);
      __syncwarp();
    }
    float s[kTok / 16][NH][4] = {};       // tokens 16 x + r8 (+ 8), heads as in o
#pragma unroll
    for (int k = 0; k < NK; k++)
      if (k < ksteps) {
#pragma unroll
        for (int x = 0; x < kTok / 16; x++) {
          uint32_t a[4];
          ldmatrix_x4(sk + (x * 16 + (lane & 15)) * pitch + (lane >> 4) * 16 + k * 32, a);
#pragma unroll
          for (int t = 0; t < NH; t++) mma_bf16(s[x][t], a, qf[k][t][0], qf[k][t][1]);
        }
      }
    float mx[NH][2];
#pragma unroll
    for (int t = 0; t < NH; t++) { mx[t][0] = m[t][0]; mx[t][1] = m[t][1]; }
#pragma unroll
    for (int x = 0; x < kTok / 16; x++)
#pragma unroll
      for (int r = 0; r < 2; r++) {
        const int tok = x * 16 + r * 8 + r8;
        float f = 1.f;
        if (!PAIR) asm volatile("ld.shared.f32 %0, [%1];" : "=f"(f) : "r"(sk + tok * pitch + p.Dp * 2) : "memory");
        const bool seen = tok < n && (!PAIR || tok >= lo - (t0 + (warp + kWarps * i) * kTok));
#pragma unroll
        for (int t = 0; t < NH; t++)
#pragma unroll
          for (int j = 0; j < 2; j++) {
            float& v = s[x][t][2 * r + j];
            v = seen ? capped_log2(PAIR ? v : v * f, p.softcap) : kNegBig;
            mx[t][j] = fmaxf(mx[t][j], v);
          }
      }
    bool grew = false;
#pragma unroll
    for (int t = 0; t < NH; t++)
#pragma unroll
      for (int j = 0; j < 2; j++) {
        mx[t][j] = fmaxf(mx[t][j], __shfl_xor_sync(0xffffffffu, mx[t][j], 4));
        mx[t][j] = fmaxf(mx[t][j], __shfl_xor_sync(0xffffffffu, mx[t][j], 8));
        mx[t][j] = fmaxf(mx[t][j], __shfl_xor_sync(0xffffffffu, mx[t][j], 16));
        grew |= mx[t][j] > m[t][j];
      }
    if (__any_sync(0xffffffffu, grew)) {
#pragma unroll
      for (int t = 0; t < NH; t++)
#pragma unroll
        for (int j = 0; j < 2; j++) {
          const float c = exp2f(m[t][j] - mx[t][j]);
          m[t][j] = mx[t][j];
          l[t][j] *= c;
#pragma unroll
          for (int k = 0; k < NK; k++) { o[k][t][j] *= c; o[k][t][2 + j] *= c; }
        }
    }
    // weights as the right operand of the sums (tokens x heads): the accumulator tiles transposed
    uint32_t w[kTok / 16][NH][2];
#pragma unroll
    for (int x = 0; x < kTok / 16; x++)
#pragma unroll
      for (int t = 0; t < NH; t++)
#pragma unroll
        for (int r = 0; r < 2; r++) {
          const float p0 = exp2f(s[x][t][2 * r] - m[t][0]), p1 = exp2f(s[x][t][2 * r + 1] - m[t][1]);
          l[t][0] += p0;
          l[t][1] += p1;
          w[x][t][r] = transpose_8x8(pack_bf16(p0, p1));
        }
#pragma unroll
    for (int k = 0; k < NK; k++)
      if (k < vsteps) {
#pragma unroll
        for (int x = 0; x < kTok / 16; x++) {
          uint32_t a[4];               // values transposed: channels x tokens
          ldmatrix_x4_trans(sk + (x * 16 + (lane & 7) + ((lane >> 4) << 3)) * pitch + voff * 2 + k * 32 + ((lane >> 3) & 1) * 16, a);
#pragma unroll
          for (int t = 0; t < NH; t++) mma_bf16(o[k][t], a, w[x][t][0], w[x][t][1]);
        }
      }
    __syncwarp();
    issue(i + kStages);
  }
  if (done < mine) {
    // gave up: let the copies in flight land before this memory goes away, and report
    for (int i = done; i < mine && i < done + kStages; i++)
      for (int spin = 0; spin < 20000 && !sm100::mbar_try_wait(smem_addr(&full[warp][i % kStages]), uint32_t(i / kStages) & 1u); spin++) __nanosleep(50);
    if (lane == 0) atomicExch(p.err, 1);
  }
#pragma unroll
  for (int t = 0; t < NH; t++)
#pragma unroll
    for (int j = 0; j < 2; j++) {
      l[t][j] += __shfl_xor_sync(0xffffffffu, l[t][j], 4);
      l[t][j] += __shfl_xor_sync(0xffffffffu, l[t][j], 8);
      l[t][j] += __shfl_xor_sync(0xffffffffu, l[t][j], 16);
      if (r8 == 0) {
        sh_m[warp][t * 8 + quad * 2 + j] = m[t][j];
        sh_l[warp][t * 8 + quad * 2 + j] = l[t][j];
      }
    }
  __syncthreads();                          // the rings are free: their space takes the warps' sums [warps][16][Vp]
  float* so = reinterpret_cast<float*>(dsm);
#pragma unroll
  for (int k = 0; k < NK; k++)
    if (k < vsteps) {
#pragma unroll
      for (int t = 0; t < NH; t++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
          const int h = t * 8 + quad * 2 + (j & 1);
          if (h < nq) so[(warp * 16 + h) * Vp + k * 16 + r8 + (j >> 1) * 8] = o[k][t][j];
        }
    }
  if (tid < NH * 8) {
    float m = kNegBig, l = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; w++) m = fmaxf(m, sh_m[w][tid]);
#pragma unroll
    for (int w = 0; w < kWarps; w++) {
      const float f = exp2f(sh_m[w][tid] - m);
      l = fmaf(sh_l[w][tid], f, l);
      sh_m[w][tid] = f;                     // factor of the warp from here on
    }
    sh_ml[tid][0] = m;
    sh_ml[tid][1] = l;
  }
  __syncthreads();
  __nv_bfloat16* out = p.out + (size_t(row) * p.heads + h0) * Vp;
  const __nv_bfloat16* gate = PAIR && p.gate ? p.gate + size_t(row) * p.ldg + size_t(h0) * Vp : nullptr;
  const int total = nq * Vp / 4;
  for (int i = tid; i < total; i += kWarps * 32) {
    const int h = i * 4 / Vp;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < kWarps; w++) {
      const float4 v = *reinterpret_cast<const float4*>(so + w * 16 * Vp + i * 4);
      const float f = sh_m[w][h];
      a.x = fmaf(v.x, f, a.x); a.y = fmaf(v.y, f, a.y); a.z = fmaf(v.z, f, a.z); a.w = fmaf(v.w, f, a.w);
    }
    if (S == 1) {
      const float l = sh_ml[h][1], f = l > 0.f ? 1.f / l : 0.f;
      a = make_float4(a.x * f, a.y * f, a.z * f, a.w * f);
      if (PAIR && gate) a = gated(a, gate + i * 4);
      *reinterpret_cast<uint2*>(out + i * 4) = make_uint2(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w));
    } else {
      *reinterpret_cast<float4*>(so + i * 4) = a;
    }
  }
  if (S == 1) return;
  cluster_sync();
  if (tid < 16 * kMaxSplits) {              // as many as there are threads
    const int r = tid >> 4, h = tid & 15;
    const uint32_t a = smem_addr(&sh_ml[h][0]);
    sh_sm[r][h] = r < S && h < nq ? ld_cluster_f32(a, r) : kNegBig;
    sh_fac[r][h] = r < S && h < nq ? ld_cluster_f32(a + 4, r) : 0.f;
  }
  __syncthreads();
  if (tid < 16) {
    float mx = kNegBig, l = 0.f;
    for (int r = 0; r < S; r++) mx = fmaxf(mx, sh_sm[r][tid]);
    for (int r = 0; r < S; r++) l = fmaf(sh_fac[r][tid], exp2f(sh_sm[r][tid] - mx), l);
    for (int r = 0; r < S; r++) sh_fac[r][tid] = l > 0.f ? exp2f(sh_sm[r][tid] - mx) / l : 0.f;
  }
  __syncthreads();
  const int per = (total + S - 1) / S;
  const uint32_t soa = smem_addr(so);
  for (int i = tid; i < per; i += kWarps * 32) {
    const int idx = sp * per + i;
    if (idx >= total) break;
    const int h = idx * 4 / Vp;
    float4 v[kMaxSplits], a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < kMaxSplits; r++)
      if (r < S) v[r] = ld_cluster_f32x4(soa + idx * 16, r);
#pragma unroll
    for (int r = 0; r < kMaxSplits; r++)
      if (r < S) {
        const float f = sh_fac[r][h];
        a.x = fmaf(v[r].x, f, a.x); a.y = fmaf(v[r].y, f, a.y); a.z = fmaf(v[r].z, f, a.z); a.w = fmaf(v[r].w, f, a.w);
      }
    if (PAIR && gate) a = gated(a, gate + idx * 4);
    *reinterpret_cast<uint2*>(out + idx * 4) = make_uint2(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w));
  }
  cluster_sync();                           // nobody leaves while a peer may still read its shared memory
}

template <int NK, int NH, int kTok, bool PAIR>
cudaError_t launch_rows(const RowsParams& p, int rows, cudaStream_t st) {
  static bool done = false;
  const int pitch = (p.Dp + (PAIR ? p.Vp : 0) + kRowPad) * 2;
  const size_t ring = size_t(kWarps) * kStages * kTok * pitch, sums = size_t(kWarps) * 16 * p.Vp * 4, smem = ring > sums ? ring : sums;
  cudaError_t e = allow_smem(k_shared_rows<NK, NH, kTok, PAIR>, smem, &done);
  const dim3 grid(rows, p.kv_heads * ((p.heads / p.kv_heads + 15) / 16), p.splits);
  return e != cudaSuccess ? e : pdl::launch(k_shared_rows<NK, NH, kTok, PAIR>, grid, dim3(kWarps * 32), smem, st, p.splits, p);
}
// with a value beside the key a row is twice as long: half as many tokens per unit keep two CTAs per SM
template <int NH, bool PAIR>
cudaError_t launch_rows(const RowsParams& p, int rows, cudaStream_t st) {
  const int d = p.Dp > p.Vp ? p.Dp : p.Vp;
  return d <= 32 ? launch_rows<2, NH, 32, PAIR>(p, rows, st) : (d <= 64 ? launch_rows<4, NH, 32, PAIR>(p, rows, st) : launch_rows<8, NH, PAIR ? 16 : 32, PAIR>(p, rows, st));
}
int clamp_splits(int s) { return s < 1 ? 1 : (s > kMaxSplits ? kMaxSplits : s); }

// ---- prefill form --------------------------------------------------------------------------------------------------------
struct PrefillParams {
  const __nv_bfloat16* q;   // [rows, ldq], head h at h * Dp
  const __nv_bfloat16* cache;
  __nv_bfloat16* out;       // [rows, ldo], head h at h * Vp
  const int* tiles;         // [ntiles, 4]: first query row, rows (<= 64), unused, keys the first row sees
  const int* seq_of_row;    // table row of a query row
  const int* tables;
  int ldq, ldo, heads, kv_heads, Dp, Vp, block_size, max_blocks;   // Vp, window, chunk, gate: as in RowsParams
  float softcap;
  int window, chunk;
  const __nv_bfloat16* gate;
  int ldg;
};

// 64 query rows of one sequence and one head per CTA, four warps of 16 rows; tiles of 64 cached rows, keys and values at once, in two
// cp.async stages.
constexpr int kPK = 64;
template <int VT, bool PAIR>
__global__ void __launch_bounds__(128, VT > 8 ? 2 : 3) k_shared_prefill_mma(const PrefillParams p) {
  extern __shared__ __align__(128) uint8_t dsm[];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int* tl = p.tiles + 4 * blockIdx.y;
  const int row0 = tl[0], nrows = tl[1], see0 = tl[3], h = blockIdx.x, g = h / (p.heads / p.kv_heads);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r8 = lane >> 2, quad = lane & 3;
  const int Vp = PAIR ? p.Vp : p.Dp, voff = PAIR ? p.Dp : 0, rowlen = p.Dp + (PAIR ? Vp : 0) + kRowPad;
  const int ksteps = p.Dp / 16, qpitch = (p.Dp + kRowPad) * 2, pitch = rowlen * 2, vblocks = Vp / 16, nch = p.Dp / 8;
  const int rch = PAIR ? (p.Dp + Vp) / 8 : nch + 1;                  // 16-byte pieces of a cached row; a factor lies in the pad
  const uint32_t sq = smem_addr(dsm), sk0 = sq + 64 * qpitch;
  const int* bt = p.tables + size_t(p.seq_of_row[row0]) * p.max_blocks;
  const int nkeys = min(see0 + nrows - 1, p.max_blocks * p.block_size), ntiles = (nkeys + kPK - 1) / kPK;
  const int first = PAIR ? first_visible(see0, p.window, p.chunk) / kPK : 0;

  // rows are copied by groups of lanes: 4 rows per warp pass, 8 lanes per row
  const int g8 = lane >> 3, l8 = lane & 7;
  for (int r = warp * 4 + g8; r < 64; r += 16) {
    const uint32_t d = sq + r * qpitch;
    const __nv_bfloat16* src = p.q + size_t(row0 + r) * p.ldq + size_t(h) * p.Dp;
    for (int c = l8; c < nch; c += 8) {
      if (r < nrows) cp_async16(d + c * 16, src + c * 8);
      else st_zero16(d + c * 16);
    }
  }
  auto issue = [&](int i) {
    if (i < ntiles) {
      const uint32_t kb = sk0 + (i & 1) * kPK * pitch;
      for (int r = warp * 4 + g8; r < kPK; r += 16) {
        const int tok = i * kPK + r;
        const uint32_t kd = kb + r * pitch;
        if (tok < nkeys) {
          const int pg = tok / p.block_size;
          const __nv_bfloat16* src = p.cache + ((size_t(bt[pg]) * p.kv_heads + g) * p.block_size + (tok - pg * p.block_size)) * rowlen;
          for (int c = l8; c < rch; c += 8) cp_async16(kd + c * 16, src + c * 8);
        } else {
          for (int c = l8; c < rch; c += 8) st_zero16(kd + c * 16);
        }
      }
    } else if (PAIR && p.gate && i == ntiles) {    // behind the last tile: the gates of these rows
      const uint32_t gb = sk0 + (i & 1) * kPK * pitch;
      for (int r = warp * 4 + g8; r < nrows; r += 16)
        for (int c = l8; c < Vp / 8; c += 8) cp_async16(gb + r * pitch + c * 16, p.gate + size_t(row0 + r) * p.ldg + size_t(h) * Vp + c * 8);
    }
    cp_async_commit();
  };
  float o[VT * 2][4];
#pragma unroll
  for (int n = 0; n < VT * 2; n++) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m_lo = kNegBig, m_hi = kNegBig, l_lo = 0.f, l_hi = 0.f;
  const int see_lo = see0 + warp * 16 + r8, see_hi = see_lo + 8;   // keys visible to this lane's two rows
  int lo_lo = 0, lo_hi = 0, lo_min = 0, lo_max = 0;                // first visible key of this lane's rows, of the warp's first and last row
  if constexpr (PAIR) {
    lo_lo = first_visible(see_lo, p.window, p.chunk);
    lo_hi = first_visible(see_hi, p.window, p.chunk);
    lo_min = first_visible(see0 + warp * 16, p.window, p.chunk);
    lo_max = first_visible(see0 + warp * 16 + 15, p.window, p.chunk);
  }
  issue(first);
  for (int i = first; i < ntiles; i++) {
    issue(i + 1);
    cp_async_wait<1>();
    __syncthreads();
    const int tok0 = i * kPK;
    if (tok0 < see0 + warp * 16 + 15 && (!PAIR || tok0 + kPK > lo_min)) {   // otherwise every key of the tile is hidden from this warp's rows
      const uint32_t sk = sk0 + (i & 1) * kPK * pitch;
      float s[kPK / 8][4];
#pragma unroll
      for (int n = 0; n < kPK / 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      const uint32_t qaddr = sq + (warp * 16 + (lane & 15)) * qpitch + (lane >> 4) * 16;
      const uint32_t kaddr = sk + ((lane & 7) + ((lane >> 4) << 3)) * pitch + ((lane >> 3) & 1) * 16;
      for (int ks = 0; ks < ksteps; ks++) {
        uint32_t a[4];
        ldmatrix_x4(qaddr + ks * 32, a);
#pragma unroll
        for (int n = 0; n < kPK / 16; n++) {
          uint32_t b[4];
          ldmatrix_x4(kaddr + n * 16 * pitch + ks * 32, b);
          mma_bf16(s[2 * n], a, b[0], b[1]);
          mma_bf16(s[2 * n + 1], a, b[2], b[3]);
        }
      }
      const bool diagonal = tok0 + kPK > see0 + warp * 16, edge = PAIR && tok0 < lo_max;
      float x_lo = m_lo, x_hi = m_hi;
#pragma unroll
      for (int n = 0; n < kPK / 8; n++)
#pragma unroll
        for (int j = 0; j < 2; j++) {
          if constexpr (PAIR) {
            s[n][j] = capped_log2(s[n][j], p.softcap);
            s[n][2 + j] = capped_log2(s[n][2 + j], p.softcap);
            if (edge) {
              const int tok = tok0 + n * 8 + quad * 2 + j;
              if (tok < lo_lo) s[n][j] = kNegBig;
              if (tok < lo_hi) s[n][2 + j] = kNegBig;
            }
          } else {
            float f;
            asm volatile("ld.shared.f32 %0, [%1];" : "=f"(f) : "r"(sk + (n * 8 + quad * 2 + j) * pitch + p.Dp * 2) : "memory");
            s[n][j] = capped_log2(s[n][j] * f, p.softcap);
            s[n][2 + j] = capped_log2(s[n][2 + j] * f, p.softcap);
          }
          if (diagonal) {
            const int tok = tok0 + n * 8 + quad * 2 + j;
            if (tok >= see_lo) s[n][j] = kNegBig;
            if (tok >= see_hi) s[n][2 + j] = kNegBig;
          }
        }
#pragma unroll
      for (int n = 0; n < kPK / 8; n++) { x_lo = fmaxf(x_lo, fmaxf(s[n][0], s[n][1])); x_hi = fmaxf(x_hi, fmaxf(s[n][2], s[n][3])); }
      x_lo = fmaxf(x_lo, __shfl_xor_sync(0xffffffffu, x_lo, 1));
      x_lo = fmaxf(x_lo, __shfl_xor_sync(0xffffffffu, x_lo, 2));
      x_hi = fmaxf(x_hi, __shfl_xor_sync(0xffffffffu, x_hi, 1));
      x_hi = fmaxf(x_hi, __shfl_xor_sync(0xffffffffu, x_hi, 2));
      const float c_lo = exp2f(m_lo - x_lo), c_hi = exp2f(m_hi - x_hi);
      m_lo = x_lo;
      m_hi = x_hi;
      float t_lo = 0.f, t_hi = 0.f;
      uint32_t pa[kPK / 16][4];
#pragma unroll
      for (int n = 0; n < kPK / 8; n++) {
        const float p0 = exp2f(s[n][0] - x_lo), p1 = exp2f(s[n][1] - x_lo), p2 = exp2f(s[n][2] - x_hi), p3 = exp2f(s[n][3] - x_hi);
        t_lo += p0 + p1;
        t_hi += p2 + p3;
        pa[n >> 1][(n & 1) * 2] = pack_bf16(p0, p1);
        pa[n >> 1][(n & 1) * 2 + 1] = pack_bf16(p2, p3);
      }
      l_lo = l_lo * c_lo + t_lo;
      l_hi = l_hi * c_hi + t_hi;
#pragma unroll
      for (int n = 0; n < VT * 2; n++) { o[n][0] *= c_lo; o[n][1] *= c_lo; o[n][2] *= c_hi; o[n][3] *= c_hi; }
#pragma unroll
      for (int b = 0; b < VT; b++) {
        if (b < vblocks) {
#pragma unroll
          for (int ks = 0; ks < kPK / 16; ks++) {
            uint32_t v[4];
            ldmatrix_x4_trans(sk + (ks * 16 + (lane & 15)) * pitch + voff * 2 + b * 32 + (lane >> 4) * 16, v);
            mma_bf16(o[2 * b], pa[ks], v[0], v[1]);
            mma_bf16(o[2 * b + 1], pa[ks], v[2], v[3]);
          }
        }
      }
    }
    __syncthreads();
  }
  cp_async_wait<0>();
  if (PAIR && p.gate) __syncthreads();
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
  const float f_lo = l_lo > 0.f ? 1.f / l_lo : 0.f, f_hi = l_hi > 0.f ? 1.f / l_hi : 0.f;
  const int rl = warp * 16 + r8, rh = rl + 8;
#pragma unroll
  for (int n = 0; n < VT * 2; n++) {
    if (n < vblocks * 2) {
      const int col = h * Vp + n * 8 + quad * 2;
      auto put = [&](int r, float a, float b) {
        if (r >= nrows) return;
        if (PAIR && p.gate) {
          const float2 gt = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(dsm + (sk0 - sq) + ((ntiles & 1) * kPK + r) * pitch + (n * 8 + quad * 2) * 2));
          a *= vec::sigmoid<__nv_bfloat16>(gt.x);
          b *= vec::sigmoid<__nv_bfloat16>(gt.y);
        }
        *reinterpret_cast<uint32_t*>(p.out + size_t(row0 + r) * p.ldo + col) = pack_bf16(a, b);
      };
      put(rl, o[n][0] * f_lo, o[n][1] * f_lo);
      put(rh, o[n][2] * f_hi, o[n][3] * f_hi);
    }
  }
}

template <int VT, bool PAIR>
cudaError_t launch_prefill(const PrefillParams& p, dim3 grid, size_t smem, cudaStream_t st) {
  static bool done = false;
  cudaError_t e = allow_smem(k_shared_prefill_mma<VT, PAIR>, smem, &done);
  return e != cudaSuccess ? e : pdl::launch(k_shared_prefill_mma<VT, PAIR>, grid, dim3(128), smem, st, 1, p);
}
template <bool PAIR>
cudaError_t launch_prefill(const PrefillParams& p, int ntiles, cudaStream_t st) {
  const size_t smem = size_t(64) * (p.Dp + kRowPad) * 2 + size_t(2) * kPK * (p.Dp + (PAIR ? p.Vp : 0) + kRowPad) * 2;
  const dim3 grid(p.heads, ntiles);
  if (p.Vp <= 32) return launch_prefill<2, PAIR>(p, grid, smem, st);
  if (p.Vp <= 64) return launch_prefill<4, PAIR>(p, grid, smem, st);
  if (p.Vp <= 128) return launch_prefill<8, PAIR>(p, grid, smem, st);
  return launch_prefill<16, PAIR>(p, grid, smem, st);
}

}  // namespace

extern "C" {

int tbv_op_shared_attn_prep(void* qk, void* qa, void* cache, const void* fold, const void* positions, const void* slots, int rows,
                            int n_rows_form, int ldq, int heads, int kv_heads, int dim, int Dp, int block_size, float eps, float temp_coef,
                            double temp_every, int bf16, void* stream) {
  if (rows <= 0) return 0;
  if (dim > Dp || dim <= 0 || (Dp % 16) || kv_heads <= 0 || heads % kv_heads || n_rows_form > rows || block_size <= 0 || !(temp_every > 0)) return -2;
  PrepParams p{qk, qa, cache, static_cast<const float*>(fold), static_cast<const int*>(positions), static_cast<const long long*>(slots),
               rows, ldq, heads, kv_heads, dim, Dp, n_rows_form, block_size, eps, temp_coef, temp_every};
  const dim3 grid(unsigned(((long long)rows * (heads + kv_heads) + 7) / 8));
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = bf16 ? pdl::launch(k_shared_prep<__nv_bfloat16>, grid, dim3(256), 0, st, 1, p) : pdl::launch(k_shared_prep<float>, grid, dim3(256), 0, st, 1, p);
  return e == cudaSuccess ? 0 : -1;
}

// qa [rows, heads, Dp + pad], cache [blocks, kv_heads, block_size, Dp + pad], softcap 0 = none; a row sees the first ctx_lens[row] tokens.
int tbv_op_shared_attn_rows(const void* qa, const void* cache, const void* tables, const void* seq_of_row, const void* ctx_lens, void* out,
                            int rows, int heads, int kv_heads, int Dp, int block_size, int max_blocks, int splits, float softcap, int bf16,
                            void* stream) {
  if (rows <= 0) return 0;
  if ((Dp % 16) || Dp <= 0 || kv_heads <= 0 || heads % kv_heads || block_size <= 0) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int *tb = static_cast<const int*>(tables), *sq = static_cast<const int*>(seq_of_row), *cl = static_cast<const int*>(ctx_lens);
  if (!bf16 || Dp > 128 || (block_size % 16))
    return tbvops::shared_attn_rows_any(qa, cache, tb, sq, cl, out, rows, heads, kv_heads, Dp, block_size, max_blocks, splits, softcap, bf16, st);
  RowsParams p{static_cast<const __nv_bfloat16*>(qa), static_cast<const __nv_bfloat16*>(cache), static_cast<__nv_bfloat16*>(out), tb, sq, cl,
               heads, kv_heads, Dp, Dp, block_size, max_blocks, clamp_splits(splits), softcap, tbvops::gemm_err_flag(), 0, 0, nullptr, 0};
  cudaError_t e = heads / kv_heads <= 8 ? launch_rows<1, false>(p, rows, st) : launch_rows<2, false>(p, rows, st);
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] shared-row attention launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

// head sizes (padded) that the prefill form takes
int tbv_op_shared_prefill_max_dim(void) { return 256; }

int tbv_op_shared_attn_prefill(const void* q, const void* cache, const void* tables, const void* seq_of_row, const void* tiles, void* out,
                               int ntiles, int ldq, int ldo, int heads, int kv_heads, int Dp, int block_size, int max_blocks, float softcap,
                               void* stream) {
  if (ntiles <= 0) return 0;
  if ((Dp % 16) || Dp > 256 || (ldq % 8) || (ldo % 8) || kv_heads <= 0 || heads % kv_heads || ntiles > 65535 || !seq_of_row) return -2;
  PrefillParams p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(cache), static_cast<__nv_bfloat16*>(out),
                  static_cast<const int*>(tiles), static_cast<const int*>(seq_of_row), static_cast<const int*>(tables),
                  ldq, ldo, heads, kv_heads, Dp, Dp, block_size, max_blocks, softcap, 0, 0, nullptr, 0};
  cudaError_t e = launch_prefill<false>(p, ntiles, static_cast<cudaStream_t>(stream));
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] shared-row prefill launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

// ---- paired rows: see the top.  Cache [blocks, kv_heads, block_size, Dp + Vp + pad]. ------------------------------------------------
// wide [rows, ldw]: queries, keys, values (kv_heads 0: queries only, nothing is written to a cache); turns [pairs] or pairs 0.
int tbv_op_paired_attn_prep(void* wide, void* qa, void* cache, const void* qn, const void* kn, const void* turns, const void* positions, const void* slots,
                            int rows, int n_rows_form, int ldw, int heads, int kv_heads, int dim, int Dp, int Vp, int pairs, int block_size, float eps, int bf16,
                            void* stream) {
  if (rows <= 0) return 0;
  if (dim > Dp || dim <= 0 || (Dp % 16) || (Vp % 16) || heads <= 0 || kv_heads < 0 || n_rows_form > rows || block_size <= 0 || (ldw % 8) || pairs < 0 || pairs > kMaxPairs ||
      2 * pairs > dim || (pairs && !turns)) return -2;
  PairPrepParams p{wide, qa, cache, static_cast<const float*>(qn), static_cast<const float*>(kn), static_cast<const float2*>(turns), static_cast<const int*>(positions),
                   static_cast<const long long*>(slots), ldw, heads, kv_heads, dim, Dp, Vp, pairs, n_rows_form, block_size, eps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = bf16 ? pdl::launch(k_paired_prep<__nv_bfloat16>, dim3(rows), dim3(256), 0, st, 1, p) : pdl::launch(k_paired_prep<float>, dim3(rows), dim3(256), 0, st, 1, p);
  return e == cudaSuccess ? 0 : -1;
}

// Norms per head without weights: wide as above; qscale [heads] fp32; v_first [rows, kv_heads * Vp] or null, lambda (device) or null: see k_head_prep.
int tbv_op_head_attn_prep(void* wide, void* qa, void* cache, const void* qscale, const void* turns, const void* positions, const void* slots, void* v_first,
                          const void* lambda, int rows, int n_rows_form, int ldw, int heads, int kv_heads, int dim, int Dp, int Vp, int pairs, int block_size,
                          float eps, int bf16, void* stream) {
  if (rows <= 0) return 0;
  if (dim > Dp || dim <= 0 || (Dp % 16) || (Vp % 16) || Vp <= 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || n_rows_form > rows || block_size <= 0 || (ldw % 8) ||
      pairs < 0 || 2 * pairs > dim || (pairs && !turns) || (lambda && !v_first)) return -2;
  HeadPrepParams p{wide, qa, cache, static_cast<const float*>(qscale), static_cast<const float2*>(turns), static_cast<const int*>(positions),
                   static_cast<const long long*>(slots), v_first, static_cast<const float*>(lambda), rows, ldw, heads, kv_heads, dim, Dp, Vp, pairs, n_rows_form,
                   block_size, eps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = bf16 ? launch_head_prep<__nv_bfloat16>(p, st) : launch_head_prep<float>(p, st);
  return e == cudaSuccess ? 0 : -1;
}

// qa [rows, heads, Dp + pad] -> out [rows, heads, Vp]; window / chunk: attn_mma::first_visible; gate [rows, ldg] or null.
int tbv_op_paired_attn_rows(const void* qa, const void* cache, const void* tables, const void* seq_of_row, const void* ctx_lens, const void* gate, void* out,
                            int rows, int heads, int kv_heads, int Dp, int Vp, int ldg, int block_size, int max_blocks, int splits, float softcap, int window, int chunk,
                            int bf16, void* stream) {
  if (rows <= 0) return 0;
  if ((Dp % 16) || (Vp % 16) || Dp <= 0 || Vp <= 0 || kv_heads <= 0 || heads % kv_heads || block_size <= 0 || (gate && (ldg % 8)) || window < 0 || chunk < 0) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int *tb = static_cast<const int*>(tables), *sq = static_cast<const int*>(seq_of_row), *cl = static_cast<const int*>(ctx_lens);
  if (!bf16 || Dp > 128 || Vp > 128 || (block_size % 16))
    return tbvops::paired_attn_rows_any(qa, cache, tb, sq, cl, gate, out, rows, heads, kv_heads, Dp, Vp, ldg, block_size, max_blocks, splits, softcap, window, chunk, bf16, st);
  RowsParams p{static_cast<const __nv_bfloat16*>(qa), static_cast<const __nv_bfloat16*>(cache), static_cast<__nv_bfloat16*>(out), tb, sq, cl,
               heads, kv_heads, Dp, Vp, block_size, max_blocks, clamp_splits(splits), softcap, tbvops::gemm_err_flag(), window, chunk,
               static_cast<const __nv_bfloat16*>(gate), ldg};
  cudaError_t e = heads / kv_heads <= 8 ? launch_rows<1, true>(p, rows, st) : launch_rows<2, true>(p, rows, st);
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] paired-row attention launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

int tbv_op_paired_prefill_fits(int Dp, int Vp) { return Vp <= 256 && size_t(64) * (Dp + kRowPad) * 2 + size_t(2) * kPK * (Dp + Vp + kRowPad) * 2 <= kMaxSmem ? 1 : 0; }

// bf16; q [rows, ldq] with head h at h * Dp, out [rows, ldo] with head h at h * Vp
int tbv_op_paired_attn_prefill(const void* q, const void* cache, const void* tables, const void* seq_of_row, const void* tiles, const void* gate, void* out,
                               int ntiles, int ldq, int ldo, int heads, int kv_heads, int Dp, int Vp, int ldg, int block_size, int max_blocks, float softcap, int window,
                               int chunk, void* stream) {
  if (ntiles <= 0) return 0;
  if ((Dp % 16) || (Vp % 16) || (ldq % 8) || (ldo % 8) || kv_heads <= 0 || heads % kv_heads || ntiles > 65535 || !seq_of_row || (gate && (ldg % 8)) || window < 0 || chunk < 0 ||
      !tbv_op_paired_prefill_fits(Dp, Vp)) return -2;
  PrefillParams p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(cache), static_cast<__nv_bfloat16*>(out),
                  static_cast<const int*>(tiles), static_cast<const int*>(seq_of_row), static_cast<const int*>(tables),
                  ldq, ldo, heads, kv_heads, Dp, Vp, block_size, max_blocks, softcap, window, chunk, static_cast<const __nv_bfloat16*>(gate), ldg};
  cudaError_t e = launch_prefill<true>(p, ntiles, static_cast<cudaStream_t>(stream));
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] paired-row prefill launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

}  // extern "C"
