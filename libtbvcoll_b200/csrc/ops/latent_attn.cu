// latent_attn.cu — attention over a compressed (latent) paged cache, with a learned sink per head.
//
// A cached token is one row of Dk = Rp + rotp values shared by all heads: the normalised latent c (R values, padded to Rp)
// and one rotated key part (padded to rotp).  Rows of the cache (and of the folded queries) lie kRowPad values apart: the tokens of
// a block come into shared memory as ONE bulk copy and already have the odd 16-byte pitch that ldmatrix wants.  Head h scores it as (q_h . W_uk,h c + q_rot,h . k_rot) * scale and its
// value is W_uv,h c.  Two forms of the same sum:
//   rows form     W_uk is folded into the query (qa_h = W_uk,h^T q_h), the cache rows serve as keys AND as values, and the
//                 result is a latent per head that W_uv expands afterwards.  The cache is read once for all heads: the
//                 decode form, and the form for portions of a few tokens.
//   prefill form  keys and values of the visible context are expanded once into dense rows and many query rows share
//                 them: a third of the arithmetic per (query, key) pair.
// Scores, softmax and sums are fp32; the denominator contains exp(sink_h) once.  With a window a row sees the last `window` keys, its own included; keys
// before the first visible one are not read.
//
// The rows form also serves attention whose values are the unnormalised keys (template KS; shared_attn.cu): kv_heads rows per token, each used by
// heads / kv_heads query heads, with one fp32 factor per row (kept in the row's pad) on its scores, and an optional soft cap.  And attention over rows that
// hold key and value side by side (kPaired; shared_attn.cu as well), with a window or chunks and a gate on the result.
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

constexpr int kMaxPairs = 512;
constexpr int kRowPad = 8;

// ---- rotation, latent norm, cache write ------------------------------------------------------------------------------
// Two parts, either may be left out: the latents of a token (key / value latent and rotated key part to the cache; the queries' latent, if there is one, is normed
// in place) and the rotated query parts.  With a query latent the queries come from a product behind the first part.
struct PrepParams {
  void* low;                // [rows, ldl]: latent (c_off), key part (k_off), query latent (cq_off), or null
  void* q;                  // [rows, ldq]: rotated parts of all heads at q_off, or null
  void* qa;                 // [n_rows_form, heads, Dk + kRowPad]: rotated query parts of the first n_rows_form rows go to column Rp
  void* cache;              // [slots, Dk + kRowPad]
  const float* gamma;       // [R]
  const float* q_gamma;     // [Rq]
  const float2* turns;      // [pairs]: turns per position, high and low part
  const int* positions;
  const long long* slots;
  int ldl, ldq, q_off, c_off, k_off, cq_off, Rq, heads, R, Rp, rotp, pairs, n_rows_form;
  float eps, mscale;        // mscale: factor on cos and sin
};

template <typename T>
__global__ void __launch_bounds__(256) k_latent_prep(const PrepParams p) {
  __shared__ float cs[kMaxPairs], sn[kMaxPairs], red[2][8];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int row = blockIdx.x, tid = threadIdx.x;
  const float pos = float(p.positions[row]);
  for (int i = tid; i < p.pairs; i += 256) {
    float s, c;
    vec::sincos_turns(pos, p.turns[i], &s, &c);
    cs[i] = c * p.mscale;
    sn[i] = s * p.mscale;
  }
  const int Dk = p.Rp + p.rotp, half = p.rotp / 2;
  if (p.low) {
    T* low = static_cast<T*>(p.low) + size_t(row) * p.ldl;
    const T* cv = low + p.c_off;
    T* cq = low + p.cq_off;
    float ss = 0.f, sq = 0.f;
    for (int i = tid; i < p.R; i += 256) { const float v = to_f(cv[i]); ss = fmaf(v, v, ss); }
    for (int i = tid; i < p.Rq; i += 256) { const float v = to_f(cq[i]); sq = fmaf(v, v, sq); }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      ss += __shfl_xor_sync(0xffffffffu, ss, o);
      sq += __shfl_xor_sync(0xffffffffu, sq, o);
    }
    if ((tid & 31) == 0) { red[0][tid >> 5] = ss; red[1][tid >> 5] = sq; }
    __syncthreads();
    float tot = 0.f, totq = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) { tot += red[0][w]; totq += red[1][w]; }
    const float r = 1.0f / sqrtf(tot / float(p.R) + p.eps);
    if (p.Rq) {
      const float rq = 1.0f / sqrtf(totq / float(p.Rq) + p.eps);
      for (int i = tid; i < p.Rq; i += 256) from_f(cq[i], to_f(cq[i]) * rq * p.q_gamma[i]);
    }
    const long long slot = p.slots[row];
    if (slot >= 0) {
      T* kc = static_cast<T*>(p.cache) + size_t(slot) * (Dk + kRowPad);
      for (int i = tid; i < p.Rp; i += 256) from_f(kc[i], i < p.R ? to_f(cv[i]) * r * p.gamma[i] : 0.f);
      const T* kr = low + p.k_off;
      for (int i = tid; i < half; i += 256) {
        const float a = to_f(kr[2 * i]), b = to_f(kr[2 * i + 1]);
        const bool rot = i < p.pairs;
        from_f(kc[p.Rp + 2 * i], rot ? a * cs[i] - b * sn[i] : a);
        from_f(kc[p.Rp + 2 * i + 1], rot ? b * cs[i] + a * sn[i] : b);
      }
    }
  } else {
    __syncthreads();
  }
  if (!p.q) return;
  const bool rows_form = row < p.n_rows_form;
  T* qr = static_cast<T*>(p.q) + size_t(row) * p.ldq + p.q_off;
  for (int j = tid; j < p.heads * half; j += 256) {
    const int h = j / half, i = j - h * half;
    const float a = to_f(qr[h * p.rotp + 2 * i]), b = to_f(qr[h * p.rotp + 2 * i + 1]);
    const bool rot = i < p.pairs;
    T* dst = rows_form ? static_cast<T*>(p.qa) + (size_t(row) * p.heads + h) * (Dk + kRowPad) + p.Rp + 2 * i : qr + h * p.rotp + 2 * i;
    from_f(dst[0], rot ? a * cs[i] - b * sn[i] : a);
    from_f(dst[1], rot ? b * cs[i] + a * sn[i] : b);
  }
}

// ---- rows form ---------------------------------------------------------------------------------------------------------
struct RowsParams {
  const void* qa;           // [rows, heads, Dk + kRowPad]
  const void* cache;        // [slots, Dk + kRowPad]
  const int* tables;        // [nseq, max_blocks]
  const int* seq_of_row;    // [rows] or null
  const int* ctx_lens;      // [rows]
  const float* sink;        // [heads] or null
  void* out;                // [rows, heads, Rp]
  int heads, R, Rp, rotp, block_size, max_blocks, splits;
  int kv_heads;             // cache rows per token: block b, head g and place t of a block at row (b * kv_heads + g) * block_size + t
  float scale_log2, scale;
  float softcap;            // 0: none (not in the latent form)
  int* err;                 // device flag: set to 1 if a wait for copies gave up
  int window, chunk;        // attn_mma::first_visible (window: not in the shared form, chunk: paired only)
  // paired rows: rotp = key columns (first), Rp = value columns (behind them)
  const void* gate;         // [rows, ldg] or null: results are multiplied by sigmoid of column h * Rp ..
  int ldg;
};
enum RowKind { kLatent, kShared, kPaired };

// fp32: one CTA per (row, head), tiles of 128 keys.  Exponents are taken of differences of natural-unit scores: a score of
// hundreds loses nothing to a multiplication by log2 e.
template <RowKind KIND>
__global__ void __launch_bounds__(128) k_latent_rows_f32(const RowsParams p) {
  extern __shared__ float sm[];
  __shared__ float red[4];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, Dk = p.Rp + p.rotp;
  const int kd = KIND == kPaired ? p.rotp : Dk, voff = KIND == kPaired ? p.rotp : 0;   // columns of the scores, first one of the values
  float* sq = sm;            // [kd]
  float* sp = sm + kd;       // [128]
  int* sl = reinterpret_cast<int*>(sp + 128);
  const float* qa = static_cast<const float*>(p.qa) + (size_t(row) * p.heads + h) * (kd + kRowPad);
  for (int i = tid; i < kd; i += 128) sq[i] = qa[i];
  const float* cache = static_cast<const float*>(p.cache);
  const int ctx = min(p.ctx_lens[row], p.max_blocks * p.block_size);
  const int* bt = p.tables + size_t(p.seq_of_row ? p.seq_of_row[row] : row) * p.max_blocks;
  const int G = p.kv_heads, g = h / (p.heads / G);
  constexpr int kAcc = 16;   // Rp <= 2048
  float o[kAcc];
#pragma unroll
  for (int k = 0; k < kAcc; k++) o[k] = 0.f;
  float m = kNegBig, l = 0.f;
  for (int t0 = KIND != kShared ? first_visible(ctx, p.window, p.chunk) : 0; t0 < ctx; t0 += 128) {
    const int n = min(128, ctx - t0);
    __syncthreads();
    float s = kNegBig;
    if (tid < n) {
      const int tok = t0 + tid, slot = (bt[tok / p.block_size] * G + g) * p.block_size + tok % p.block_size;
      sl[tid] = slot;
      const float4* kr = reinterpret_cast<const float4*>(cache + size_t(slot) * (Dk + kRowPad));
      const float4* q4 = reinterpret_cast<const float4*>(sq);
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int i = 0; i < kd / 4; i++) {
        const float4 k = kr[i], q = q4[i];
        a.x = fmaf(q.x, k.x, a.x); a.y = fmaf(q.y, k.y, a.y); a.z = fmaf(q.z, k.z, a.z); a.w = fmaf(q.w, k.w, a.w);
      }
      s = ((a.x + a.y) + (a.z + a.w)) * p.scale;
      if (KIND == kShared) s *= cache[size_t(slot) * (Dk + kRowPad) + Dk];
      if (KIND != kLatent && p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
    }
    float mx = s;
#pragma unroll
    for (int d = 16; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
    if ((tid & 31) == 0) red[tid >> 5] = mx;
    __syncthreads();
    const float mn = fmaxf(m, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
    const float pr = tid < n ? expf(s - mn) : 0.f, corr = expf(m - mn);
    sp[tid] = pr;
    float ps = pr;
#pragma unroll
    for (int d = 16; d > 0; d >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, d);
    __syncthreads();
    if ((tid & 31) == 0) red[tid >> 5] = ps;
    __syncthreads();
    l = l * corr + (red[0] + red[1] + red[2] + red[3]);
    m = mn;
#pragma unroll
    for (int k = 0; k < kAcc; k++) {
      const int d = tid + k * 128;
      if (d < p.R) {
        float acc = 0.f;
        for (int t = 0; t < n; t++) acc = fmaf(sp[t], cache[size_t(sl[t]) * (Dk + kRowPad) + voff + d], acc);
        o[k] = fmaf(o[k], corr, acc);
      }
    }
  }
  float c = 1.f;
  if (p.sink) {
    const float sk = p.sink[h], mf = fmaxf(m, sk);
    c = expf(m - mf);
    l = l * c + expf(sk - mf);
  }
  float* out = static_cast<float*>(p.out) + (size_t(row) * p.heads + h) * p.Rp;
#pragma unroll
  for (int k = 0; k < kAcc; k++) {
    const int d = tid + k * 128;
    if (d < p.Rp) {
      float v = d < p.R && l > 0.f ? o[k] * c / l : 0.f;
      if (KIND == kPaired && p.gate) v *= vec::sigmoid<float>(static_cast<const float*>(p.gate)[size_t(row) * p.ldg + size_t(h) * p.Rp + d]);
      out[d] = v;
    }
  }
}

// bf16: 16 heads of one row per CTA on tensor cores.  Eight warps share tiles of TT cached tokens that a ninth brings into two stages by
// bulk copies.  Scores: warp w takes tokens 8w.. of the tile over all Dk columns.  Weighted sum: it takes the latent columns of the
// 16-column blocks w, w + 8, .. (CBW of them).  grid (rows, head tiles, splits), cluster (1, 1, splits): the CTAs of a cluster cover
// disjoint token ranges and merge in split order.
constexpr int kRW = 8;
constexpr int kMaxSplits = 8;
template <int CBW, int TT, RowKind KIND>
__global__ void __launch_bounds__(kRW * 32 + 32, 1) k_latent_rows_mma(const RowsParams p) {
  extern __shared__ __align__(128) uint8_t dsm[];
  __shared__ float sh_max[kRW][16], sh_l[kRW][16], sh_ml[16][2], sh_fac[kMaxSplits][16], sh_sm[kMaxSplits][16];
  __shared__ __align__(16) uint8_t sh_p[16 * (TT * 2 + 16)];
  __shared__ unsigned long long full[2];
  __shared__ int abort_flag;
  pdl::launch_dependents();
  if (threadIdx.x == 0) {
    sm100::mbar_init(smem_addr(&full[0]), 1);
    sm100::mbar_init(smem_addr(&full[1]), 1);
    abort_flag = 0;
    sm100::mbar_fence_init();
  }
  __syncthreads();
  pdl::grid_dependency_wait();
  const int row = blockIdx.x, sp = blockIdx.z, S = p.splits;
  // head tile: 16 query heads of one cache head g
  constexpr bool HEADS = KIND != kLatent;
  const int G = HEADS ? p.kv_heads : 1, hpk = p.heads / G, tpg = (hpk + 15) / 16, g = HEADS ? blockIdx.y / tpg : 0;
  const int h0 = g * hpk + (blockIdx.y - g * tpg) * 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r8 = lane >> 2, quad = lane & 3;
  const int Dk = p.Rp + p.rotp, kd = KIND == kPaired ? p.rotp : Dk, voff = KIND == kPaired ? p.rotp : 0;   // columns: all, of the scores, before the values
  const int chunks = Dk / 8, pitch = (Dk + kRowPad) * 2, qpitch = (kd + kRowPad) * 2, ksteps = kd / 16, cblocks = p.Rp / 16;
  const uint32_t sq = smem_addr(dsm), sk0 = sq + 16 * pitch, stage = uint32_t(TT) * pitch, spb = smem_addr(sh_p);
  constexpr int kPP = TT * 2 + 16;
  const int ctx = min(p.ctx_lens[row], p.max_blocks * p.block_size);
  const int* bt = p.tables + size_t(p.seq_of_row ? p.seq_of_row[row] : row) * p.max_blocks;
  const int lo = KIND != kShared ? first_visible(ctx, p.window, p.chunk) : 0, from = lo & ~15;
  int chunk = (ctx - from + S - 1) / S;
  chunk = (chunk + 15) / 16 * 16;
  const int t0 = min(ctx, from + sp * chunk), t1 = min(ctx, t0 + chunk);
  const int ntiles = (t1 - t0 + TT - 1) / TT;

  const __nv_bfloat16* qa = static_cast<const __nv_bfloat16*>(p.qa) + (size_t(row) * p.heads + h0) * (kd + kRowPad);
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(p.cache);
  const int nq = min(16, (g + 1) * hpk - h0);
  for (int r = nq + warp; r < 16; r += kRW + 1)
    for (int c = lane; c < kd / 8; c += 32) st_zero16(sq + r * qpitch + c * 16);
  // The ninth warp brings the tiles in.  Tile i: its tokens, a block (or the part of one inside the tile) per copy, and the query rows
  // with tile 0.  A partial tile ends at a multiple of 16 tokens; its missing rows are zeros, so that a weight of zero meets no stale
  // bit pattern.  Table entries are looked up a tile ahead of their use: table and cache are two memory round trips, and both would
  // otherwise stand between two tiles.
  const int bs = p.block_size;
  auto look_up = [&](int i) {
    const int pg = (t0 + i * TT) / bs + lane;
    return pg * bs < t1 ? bt[pg] : 0;
  };
  auto issue = [&](int i, int block) {
    if (i >= ntiles) return;
    const uint32_t dst = sk0 + (i & 1) * stage, bar = smem_addr(&full[i & 1]);
    const int tok0 = t0 + i * TT, n = min(TT, t1 - tok0), pg0 = tok0 / bs;
    if (lane == 0) {
      sm100::mbar_expect_tx(bar, uint32_t(n) * uint32_t(pitch) + (i == 0 ? uint32_t(nq) * uint32_t(qpitch) : 0u));
      if (i == 0) sm100::bulk_load(sq, qa, uint32_t(nq) * qpitch, bar);
    }
    __syncwarp();
    for (int pg = pg0 + lane; pg * bs < tok0 + n; pg += 32) {
      if (pg >= pg0 + 32) block = bt[pg];      // blocks of one or two tokens only
      const int a = max(tok0, pg * bs), e = min(tok0 + n, (pg + 1) * bs);
      sm100::bulk_load(dst + (a - tok0) * pitch, cache + ((size_t(block) * G + g) * bs + (a - pg * bs)) * (Dk + kRowPad), uint32_t(e - a) * pitch, bar);
    }
    for (int r = n; r < ((n + 15) & ~15); r++)
      for (int c = lane; c < chunks; c += 32) st_zero16(dst + r * pitch + c * 16);
  };
  const bool producer = warp == kRW;
  float o[CBW][2][4];
#pragma unroll
  for (int b = 0; b < CBW; b++)
#pragma unroll
    for (int n = 0; n < 2; n++) o[b][n][0] = o[b][n][1] = o[b][n][2] = o[b][n][3] = 0.f;
  float m_lo = kNegBig, m_hi = kNegBig, l_lo = 0.f, l_hi = 0.f;
  int block = 0;
  if (producer) {
    const int block0 = look_up(0), block1 = look_up(1);
    block = look_up(2);
    issue(0, block0);
    issue(1, block1);
  }
  __syncthreads();                               // rows of zeros are in place
  for (int i = 0; i < ntiles; i++) {
    if (producer) {                              // keeps step with the barriers below, then refills the stage they released
      __syncthreads();
      __syncthreads();
      __syncthreads();
      issue(i + 2, block);
      block = look_up(i + 3);
      continue;
    }
    // zeros for a tile are stored two iterations, hence barriers, before it is read
    sm100::mbar_wait(smem_addr(&full[i & 1]), uint32_t(i >> 1) & 1u, &abort_flag, 2000000000ull);
    __syncwarp();
    const uint32_t sk = sk0 + (i & 1) * stage;
    float sc[4] = {0.f, 0.f, 0.f, 0.f}, sd[4] = {0.f, 0.f, 0.f, 0.f};
    const int n16 = (min(TT, t1 - t0 - i * TT) + 15) & ~15;
    const bool has_s = warp * 8 < n16;
    if (has_s) {
      // operands of the next two k steps are requested before the products of these two; four accumulators in turn
      const uint32_t qaddr = sq + (lane & 15) * qpitch + (lane >> 4) * 16;
      const uint32_t kaddr = sk + (warp * 8 + (lane & 7)) * pitch + (lane >> 3) * 16;
      float se[4] = {0.f, 0.f, 0.f, 0.f}, sf[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t a[2][2][4], b[2][4];
      auto load = [&](int ks, int w) {
        ldmatrix_x4(kaddr + ks * 32, b[w]);
        ldmatrix_x4(qaddr + ks * 32, a[w][0]);
        ldmatrix_x4(qaddr + ks * 32 + 32, a[w][1]);
      };
      const int pairs = ksteps / 2;
      if (pairs > 0) load(0, 0);
      int k2 = 0;
      for (; k2 + 1 < pairs; k2 += 2) {
        load(2 * k2 + 2, 1);
        mma_bf16(sc, a[0][0], b[0][0], b[0][1]);
        mma_bf16(sd, a[0][1], b[0][2], b[0][3]);
        if (k2 + 2 < pairs) load(2 * k2 + 4, 0);
        mma_bf16(se, a[1][0], b[1][0], b[1][1]);
        mma_bf16(sf, a[1][1], b[1][2], b[1][3]);
      }
      if (k2 < pairs) {
        mma_bf16(sc, a[0][0], b[0][0], b[0][1]);
        mma_bf16(sd, a[0][1], b[0][2], b[0][3]);
      }
      if (ksteps & 1) {
        const int ks = ksteps - 1;
        ldmatrix_x4(qaddr + ks * 32, a[0][0]);
        ldmatrix_x2(sk + (warp * 8 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 16 + ks * 32, b[0]);
        mma_bf16(se, a[0][0], b[0][0], b[0][1]);
      }
#pragma unroll
      for (int j = 0; j < 4; j++) sc[j] += se[j], sd[j] += sf[j];
      const int tok = t0 + i * TT + warp * 8 + quad * 2;
      if constexpr (KIND == kPaired) {
#pragma unroll
        for (int j = 0; j < 4; j++) sc[j] = tok + (j & 1) < t1 && tok + (j & 1) >= lo ? capped_log2(sc[j] + sd[j], p.softcap) : kNegBig;
      } else if constexpr (KIND == kShared) {
        float f[2];            // the two tokens' factors (stale past the end: masked below)
#pragma unroll
        for (int j = 0; j < 2; j++) asm volatile("ld.shared.f32 %0, [%1];" : "=f"(f[j]) : "r"(sk + (warp * 8 + quad * 2 + j) * pitch + Dk * 2) : "memory");
#pragma unroll
        for (int j = 0; j < 4; j++) sc[j] = tok + (j & 1) < t1 ? capped_log2((sc[j] + sd[j]) * (f[j & 1] * p.scale), p.softcap) : kNegBig;
      } else {
#pragma unroll
        for (int j = 0; j < 4; j++) sc[j] = tok + (j & 1) < t1 && tok + (j & 1) >= lo ? (sc[j] + sd[j]) * p.scale_log2 : kNegBig;
      }
      float x_lo = fmaxf(sc[0], sc[1]), x_hi = fmaxf(sc[2], sc[3]);
      x_lo = fmaxf(x_lo, __shfl_xor_sync(0xffffffffu, x_lo, 1));
      x_lo = fmaxf(x_lo, __shfl_xor_sync(0xffffffffu, x_lo, 2));
      x_hi = fmaxf(x_hi, __shfl_xor_sync(0xffffffffu, x_hi, 1));
      x_hi = fmaxf(x_hi, __shfl_xor_sync(0xffffffffu, x_hi, 2));
      if (quad == 0) { sh_max[warp][r8] = x_lo; sh_max[warp][r8 + 8] = x_hi; }
    } else if (quad == 0) {
      sh_max[warp][r8] = sh_max[warp][r8 + 8] = kNegBig;
    }
    __syncthreads();
    float n_lo = m_lo, n_hi = m_hi;
#pragma unroll
    for (int w = 0; w < TT / 8; w++) { n_lo = fmaxf(n_lo, sh_max[w][r8]); n_hi = fmaxf(n_hi, sh_max[w][r8 + 8]); }
    const float c_lo = exp2f(m_lo - n_lo), c_hi = exp2f(m_hi - n_hi);
    m_lo = n_lo;
    m_hi = n_hi;
    l_lo *= c_lo;
    l_hi *= c_hi;
    if (has_s) {
      const float p0 = exp2f(sc[0] - n_lo), p1 = exp2f(sc[1] - n_lo), p2 = exp2f(sc[2] - n_hi), p3 = exp2f(sc[3] - n_hi);
      l_lo += p0 + p1;
      l_hi += p2 + p3;
      *reinterpret_cast<uint32_t*>(sh_p + r8 * kPP + (warp * 8 + quad * 2) * 2) = pack_bf16(p0, p1);
      *reinterpret_cast<uint32_t*>(sh_p + (r8 + 8) * kPP + (warp * 8 + quad * 2) * 2) = pack_bf16(p2, p3);
    }
    __syncthreads();
#pragma unroll
    for (int b = 0; b < CBW; b++)
#pragma unroll
      for (int n = 0; n < 2; n++) { o[b][n][0] *= c_lo; o[b][n][1] *= c_lo; o[b][n][2] *= c_hi; o[b][n][3] *= c_hi; }
    uint32_t pa[2][4], v[2][CBW][4];
    auto load_v = [&](int ks, int w) {
      ldmatrix_x4(spb + (lane & 15) * kPP + (lane >> 4) * 16 + ks * 32, pa[w]);
#pragma unroll
      for (int b = 0; b < CBW; b++)
        if (warp + b * kRW < cblocks)
          ldmatrix_x4_trans(sk + (ks * 16 + (lane & 15)) * pitch + (warp + b * kRW) * 32 + voff * 2 + (lane >> 4) * 16, v[w][b]);
    };
    load_v(0, 0);
#pragma unroll
    for (int ks = 0; ks < TT / 16; ks++) {
      if (ks * 16 >= n16) break;
      if (ks + 1 < TT / 16 && ks * 16 + 16 < n16) load_v(ks + 1, (ks + 1) & 1);
#pragma unroll
      for (int b = 0; b < CBW; b++)
        if (warp + b * kRW < cblocks) {
          mma_bf16(o[b][0], pa[ks & 1], v[ks & 1][b][0], v[ks & 1][b][1]);
          mma_bf16(o[b][1], pa[ks & 1], v[ks & 1][b][2], v[ks & 1][b][3]);
        }
    }
    __syncthreads();   // this stage may be refilled
  }
  if (abort_flag && tid == 0) {
    // gave up: let the copies in flight land before this memory goes away, and report
    for (int k = 0; k < 2; k++)
      for (int spin = 0; spin < 20000 && ntiles > k && !sm100::mbar_try_wait(smem_addr(&full[k]), uint32_t((ntiles - 1 - k) >> 1) & 1u); spin++) __nanosleep(50);
    atomicExch(p.err, 1);
  }
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
  if (quad == 0 && !producer) { sh_l[warp][r8] = l_lo; sh_l[warp][r8 + 8] = l_hi; }
  if (warp == 0 && quad == 0) { sh_ml[r8][0] = m_lo; sh_ml[r8 + 8][0] = m_hi; }
  __syncthreads();     // also: every warp is done with the tiles, whose space now takes the partial results
  float* so = reinterpret_cast<float*>(dsm);   // [16][Rp]
#pragma unroll
  for (int b = 0; b < CBW; b++) {
    const int cb = warp + b * kRW;
    if (cb < cblocks && !producer) {
#pragma unroll
      for (int n = 0; n < 2; n++) {
        const int col = cb * 16 + n * 8 + quad * 2;
        *reinterpret_cast<float2*>(so + r8 * p.Rp + col) = make_float2(o[b][n][0], o[b][n][1]);
        *reinterpret_cast<float2*>(so + (r8 + 8) * p.Rp + col) = make_float2(o[b][n][2], o[b][n][3]);
      }
    }
  }
  if (tid < 16) {
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < kRW; w++) l += sh_l[w][tid];
    sh_ml[tid][1] = l;
  }
  if (S > 1) cluster_sync();
  else __syncthreads();
  // factor of every split's partial sum, the sink and the division included; all remote values are requested before one is used
  if (tid < 16 * kMaxSplits) {
    const int r = tid >> 4, h = tid & 15;
    float m = kNegBig, l = 0.f;
    if (r < S) {
      const uint32_t a = smem_addr(&sh_ml[h][0]);
      m = S > 1 ? ld_cluster_f32(a, r) : sh_ml[h][0];
      l = S > 1 ? ld_cluster_f32(a + 4, r) : sh_ml[h][1];
    }
    sh_sm[r][h] = m;
    sh_fac[r][h] = l;
  }
  __syncthreads();
  if (tid < 16) {
    const float sk = p.sink && tid < nq ? p.sink[h0 + tid] * kLog2e : kNegBig;
    float mx = sk, l = 0.f;
    for (int r = 0; r < S; r++) mx = fmaxf(mx, sh_sm[r][tid]);
    for (int r = 0; r < S; r++) l = fmaf(sh_fac[r][tid], exp2f(sh_sm[r][tid] - mx), l);
    if (p.sink) l += exp2f(sk - mx);
    for (int r = 0; r < S; r++) sh_fac[r][tid] = l > 0.f ? exp2f(sh_sm[r][tid] - mx) / l : 0.f;
  }
  __syncthreads();
  const int total = nq * p.Rp / 4, per = (total + S - 1) / S;
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (size_t(row) * p.heads + h0) * p.Rp;
  const uint32_t soa = smem_addr(so);
  for (int i = tid; i < per; i += kRW * 32 + 32) {
    const int idx = sp * per + i;
    if (idx < total) {
      const int h = idx * 4 / p.Rp;
      float4 v[kMaxSplits], a = make_float4(0.f, 0.f, 0.f, 0.f);
      if (S > 1) {
#pragma unroll
        for (int r = 0; r < kMaxSplits; r++)
          if (r < S) v[r] = ld_cluster_f32x4(soa + idx * 16, r);
      } else {
        v[0] = *reinterpret_cast<const float4*>(so + idx * 4);
      }
#pragma unroll
      for (int r = 0; r < kMaxSplits; r++)
        if (r < S) {
          const float f = sh_fac[r][h];
          a.x = fmaf(v[r].x, f, a.x); a.y = fmaf(v[r].y, f, a.y); a.z = fmaf(v[r].z, f, a.z); a.w = fmaf(v[r].w, f, a.w);
        }
      if (KIND == kPaired && p.gate) {
        const float4 gt = load_bf16x4(static_cast<const __nv_bfloat16*>(p.gate) + size_t(row) * p.ldg + size_t(h0) * p.Rp + idx * 4);
        a.x *= vec::sigmoid<__nv_bfloat16>(gt.x); a.y *= vec::sigmoid<__nv_bfloat16>(gt.y);
        a.z *= vec::sigmoid<__nv_bfloat16>(gt.z); a.w *= vec::sigmoid<__nv_bfloat16>(gt.w);
      }
      *reinterpret_cast<uint2*>(out + idx * 4) = make_uint2(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w));
    }
  }
  if (S > 1) cluster_sync();   // nobody leaves while a peer may still read its shared memory
}

// ---- prefill form --------------------------------------------------------------------------------------------------------
// cache rows of the visible context -> dense latents [n, Rp] and rotated key parts [n, rotp]
__global__ void __launch_bounds__(256) k_latent_gather(const uint4* __restrict__ cache, const long long* __restrict__ slots, uint4* c, uint4* kr,
                                                       int n, int cu, int ku) {
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int w = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (w >= n) return;
  const uint4* src = cache + size_t(slots[w]) * (cu + ku + kRowPad / 8);
  for (int i = lane; i < cu + ku; i += 32) {
    const uint4 v = src[i];
    if (i < cu) c[size_t(w) * cu + i] = v;
    else kr[size_t(w) * ku + i - cu] = v;
  }
}

struct PrefillParams {
  const __nv_bfloat16 *q, *kv, *kr;   // q [rows, ldq]; kv [ctx rows, ldkv]: keys at h * dimp, values at v_off + h * vdp; kr [ctx rows, rotp]
  __nv_bfloat16* out;                 // [rows, ldo], head h at h * vdp
  const int* tiles;                   // [ntiles, 4]: first query row, rows (<= 64), first dense context row, keys the first row sees
  const float* sink;
  int ldq, q_rot_off, ldkv, v_off, ldo, dimp, rotp, vdp;
  float scale_log2;
  int window;                         // a row sees the last `window` keys (0: all)
};

// 64 query rows of one sequence and one head per CTA, four warps of 16 rows; key / value tiles of 64 tokens in two cp.async stages.
constexpr int kPK = 64;
template <int VT>
__global__ void __launch_bounds__(128, 2) k_latent_prefill_mma(const PrefillParams p) {
  extern __shared__ __align__(128) uint8_t dsm[];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int* tl = p.tiles + 4 * blockIdx.y;
  const int row0 = tl[0], nrows = tl[1], ctx0 = tl[2], see0 = tl[3], h = blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r8 = lane >> 2, quad = lane & 3;
  const int Dq = p.dimp + p.rotp, ksteps = Dq / 16, pq = Dq * 2 + 16, pv = p.vdp * 2 + 16, vblocks = p.vdp / 16;
  const uint32_t sq = smem_addr(dsm), sk0 = sq + 64 * pq, sv0 = sk0 + 2 * kPK * pq;
  const int nkeys = see0 + nrows - 1, ntiles = (nkeys + kPK - 1) / kPK, first = first_visible(see0, p.window, 0) / kPK;
  const int nch = p.dimp / 8, rch = p.rotp / 8, vch = p.vdp / 8;

  // rows are copied by groups of lanes: 4 rows per warp pass, 8 lanes per row
  const int g8 = lane >> 3, l8 = lane & 7;
  for (int r = warp * 4 + g8; r < 64; r += 16) {
    const uint32_t d = sq + r * pq;
    if (r < nrows) {
      const __nv_bfloat16* src = p.q + size_t(row0 + r) * p.ldq;
      for (int c = l8; c < nch; c += 8) cp_async16(d + c * 16, src + h * p.dimp + c * 8);
      for (int c = l8; c < rch; c += 8) cp_async16(d + (nch + c) * 16, src + p.q_rot_off + h * p.rotp + c * 8);
    } else {
      for (int c = l8; c < nch + rch; c += 8) st_zero16(d + c * 16);
    }
  }
  auto issue = [&](int i) {
    if (i < ntiles) {
      const uint32_t kb = sk0 + (i & 1) * kPK * pq, vb = sv0 + (i & 1) * kPK * pv;
      for (int r = warp * 4 + g8; r < kPK; r += 16) {
        const int tok = i * kPK + r;
        const uint32_t kd = kb + r * pq, vd = vb + r * pv;
        if (tok < nkeys) {
          const __nv_bfloat16* src = p.kv + (long long)(ctx0 + tok) * p.ldkv;
          const __nv_bfloat16* srk = p.kr + (long long)(ctx0 + tok) * p.rotp;
          for (int c = l8; c < nch; c += 8) cp_async16(kd + c * 16, src + h * p.dimp + c * 8);
          for (int c = l8; c < rch; c += 8) cp_async16(kd + (nch + c) * 16, srk + c * 8);
          for (int c = l8; c < vch; c += 8) cp_async16(vd + c * 16, src + p.v_off + h * p.vdp + c * 8);
        } else {
          for (int c = l8; c < nch + rch; c += 8) st_zero16(kd + c * 16);
          for (int c = l8; c < vch; c += 8) st_zero16(vd + c * 16);
        }
      }
    }
    cp_async_commit();
  };
  float o[VT * 2][4];
#pragma unroll
  for (int n = 0; n < VT * 2; n++) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m_lo = kNegBig, m_hi = kNegBig, l_lo = 0.f, l_hi = 0.f;
  const int see_lo = see0 + warp * 16 + r8, see_hi = see_lo + 8;   // keys visible to this lane's two rows
  const int lo_lo = first_visible(see_lo, p.window, 0), lo_hi = first_visible(see_hi, p.window, 0);
  const int lo_min = first_visible(see0 + warp * 16, p.window, 0), lo_max = first_visible(see0 + warp * 16 + 15, p.window, 0);   // of the warp's first and last row
  issue(first);
  for (int i = first; i < ntiles; i++) {
    issue(i + 1);
    cp_async_wait<1>();
    __syncthreads();
    const int tok0 = i * kPK;
    if (tok0 < see0 + warp * 16 + 15 && tok0 + kPK > lo_min) {          // otherwise every key of the tile is hidden from this warp's rows
      const uint32_t sk = sk0 + (i & 1) * kPK * pq, sv = sv0 + (i & 1) * kPK * pv;
      float s[kPK / 8][4];
#pragma unroll
      for (int n = 0; n < kPK / 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      const uint32_t qaddr = sq + (warp * 16 + (lane & 15)) * pq + (lane >> 4) * 16;
      const uint32_t kaddr = sk + ((lane & 7) + ((lane >> 4) << 3)) * pq + ((lane >> 3) & 1) * 16;
      for (int ks = 0; ks < ksteps; ks++) {
        uint32_t a[4];
        ldmatrix_x4(qaddr + ks * 32, a);
#pragma unroll
        for (int n = 0; n < kPK / 16; n++) {
          uint32_t b[4];
          ldmatrix_x4(kaddr + n * 16 * pq + ks * 32, b);
          mma_bf16(s[2 * n], a, b[0], b[1]);
          mma_bf16(s[2 * n + 1], a, b[2], b[3]);
        }
      }
      float x_lo = m_lo, x_hi = m_hi;
      if (tok0 + kPK > see0 + warp * 16 || tok0 < lo_max) {       // the diagonal, or the window's edge
#pragma unroll
        for (int n = 0; n < kPK / 8; n++)
#pragma unroll
          for (int j = 0; j < 2; j++) {
            const int tok = tok0 + n * 8 + quad * 2 + j;
            s[n][j] = tok < see_lo && tok >= lo_lo ? s[n][j] * p.scale_log2 : kNegBig;
            s[n][2 + j] = tok < see_hi && tok >= lo_hi ? s[n][2 + j] * p.scale_log2 : kNegBig;
          }
      } else {
#pragma unroll
        for (int n = 0; n < kPK / 8; n++)
#pragma unroll
          for (int j = 0; j < 4; j++) s[n][j] *= p.scale_log2;
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
            ldmatrix_x4_trans(sv + (ks * 16 + (lane & 15)) * pv + b * 32 + (lane >> 4) * 16, v);
            mma_bf16(o[2 * b], pa[ks], v[0], v[1]);
            mma_bf16(o[2 * b + 1], pa[ks], v[2], v[3]);
          }
        }
      }
    }
    __syncthreads();
  }
  cp_async_wait<0>();
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
  float f_lo = 1.f, f_hi = 1.f;
  if (p.sink) {
    const float sk = p.sink[h] * kLog2e, x_lo = fmaxf(m_lo, sk), x_hi = fmaxf(m_hi, sk);
    f_lo = exp2f(m_lo - x_lo);
    f_hi = exp2f(m_hi - x_hi);
    l_lo = l_lo * f_lo + exp2f(sk - x_lo);
    l_hi = l_hi * f_hi + exp2f(sk - x_hi);
  }
  f_lo = l_lo > 0.f ? f_lo / l_lo : 0.f;
  f_hi = l_hi > 0.f ? f_hi / l_hi : 0.f;
  const int rl = warp * 16 + r8, rh = rl + 8;
#pragma unroll
  for (int n = 0; n < VT * 2; n++) {
    if (n < vblocks * 2) {
      const int col = h * p.vdp + n * 8 + quad * 2;
      if (rl < nrows) *reinterpret_cast<uint32_t*>(p.out + size_t(row0 + rl) * p.ldo + col) = pack_bf16(o[n][0] * f_lo, o[n][1] * f_lo);
      if (rh < nrows) *reinterpret_cast<uint32_t*>(p.out + size_t(row0 + rh) * p.ldo + col) = pack_bf16(o[n][2] * f_hi, o[n][3] * f_hi);
    }
  }
}

template <int CBW, int TT, RowKind KIND>
cudaError_t launch_rows(const RowsParams& p, dim3 grid, size_t smem, cudaStream_t st) {
  static bool done = false;
  cudaError_t e = allow_smem(k_latent_rows_mma<CBW, TT, KIND>, smem, &done);
  return e != cudaSuccess ? e : pdl::launch(k_latent_rows_mma<CBW, TT, KIND>, grid, dim3(kRW * 32 + 32), smem, st, p.splits, p);
}
template <int VT>
cudaError_t launch_prefill(const PrefillParams& p, dim3 grid, size_t smem, cudaStream_t st) {
  static bool done = false;
  cudaError_t e = allow_smem(k_latent_prefill_mma<VT>, smem, &done);
  return e != cudaSuccess ? e : pdl::launch(k_latent_prefill_mma<VT>, grid, dim3(128), smem, st, 1, p);
}
size_t rows_smem(int Dk, int TT) { return size_t(16 + 2 * TT) * (Dk * 2 + 16); }
size_t prefill_smem(int Dq, int vdp) { return size_t(64 + 2 * kPK) * (Dq * 2 + 16) + size_t(2) * kPK * (vdp * 2 + 16); }

template <RowKind KIND>
int rows_form(RowsParams& p, int rows, int bf16, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (p.heads <= 0 || p.block_size <= 0) return -2;
  p.err = tbvops::gemm_err_flag();
  cudaError_t e;
  if (!bf16) {
    p.splits = 1;
    if (p.Rp > 2048) return -2;
    e = pdl::launch(k_latent_rows_f32<KIND>, dim3(rows, p.heads), dim3(128), size_t(p.Rp + p.rotp + 256) * 4, st, 1, p);
    return e == cudaSuccess ? 0 : -1;
  }
  p.splits = p.splits < 1 ? 1 : (p.splits > kMaxSplits ? kMaxSplits : p.splits);
  const int Dk = p.Rp + p.rotp;
  const dim3 grid(rows, p.kv_heads * ((p.heads / p.kv_heads + 15) / 16), p.splits);
  const size_t s64 = rows_smem(Dk, 64), s32 = rows_smem(Dk, 32);   // either holds the [16][Rp] fp32 partials too
  if (p.Rp <= 128) e = launch_rows<1, 64, KIND>(p, grid, s64, st);
  else if (p.Rp <= 256) e = launch_rows<2, 64, KIND>(p, grid, s64, st);
  else if (p.Rp <= 512 && s64 <= kMaxSmem - 8192) e = launch_rows<4, 64, KIND>(p, grid, s64, st);
  else if (p.Rp <= 1024 && s32 <= kMaxSmem - 8192) e = launch_rows<8, 32, KIND>(p, grid, s32, st);
  else return -2;
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] latent attention launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

}  // namespace

namespace tbvops {
int shared_attn_rows_any(const void* qa, const void* cache, const int* tables, const int* seq_of_row, const int* ctx_lens, void* out, int rows,
                         int heads, int kv_heads, int Dp, int block_size, int max_blocks, int splits, float softcap, int bf16, cudaStream_t st) {
  RowsParams p{qa, cache, tables, seq_of_row, ctx_lens, nullptr, out, heads, Dp, Dp, 0, block_size, max_blocks, splits, kv_heads, kLog2e, 1.f, softcap, nullptr, 0, 0, nullptr, 0};
  return rows_form<kShared>(p, rows, bf16, st);
}
int paired_attn_rows_any(const void* qa, const void* cache, const int* tables, const int* seq_of_row, const int* ctx_lens, const void* gate, void* out, int rows,
                         int heads, int kv_heads, int Dp, int Vp, int ldg, int block_size, int max_blocks, int splits, float softcap, int window, int chunk, int bf16,
                         cudaStream_t st) {
  RowsParams p{qa, cache, tables, seq_of_row, ctx_lens, nullptr, out, heads, Vp, Vp, Dp, block_size, max_blocks, splits, kv_heads, kLog2e, 1.f, softcap, nullptr,
               window, chunk, gate, ldg};
  return rows_form<kPaired>(p, rows, bf16, st);
}
}  // namespace tbvops

extern "C" {

// low [rows, ldl] or null (then q only); q [rows, ldq] or null; Rq 0: no query latent.
int tbv_op_latent_prep(void* low, void* q, void* qa, void* cache, const void* gamma, const void* q_gamma, const void* turns, const void* positions, const void* slots,
                       int rows, int n_rows_form, int ldl, int ldq, int q_off, int c_off, int k_off, int cq_off, int Rq, int heads, int R, int Rp, int rotp, int pairs,
                       float eps, float mscale, int bf16, void* stream) {
  if (rows <= 0) return 0;
  if (pairs > kMaxPairs || pairs * 2 > rotp || R > Rp || (Rp % 16) || (rotp % 16) || n_rows_form > rows || Rq < 0 || (Rq && !q_gamma) || (low && (!cache || !slots))) return -2;
  PrepParams p{low, q, qa, cache, static_cast<const float*>(gamma), static_cast<const float*>(q_gamma), static_cast<const float2*>(turns), static_cast<const int*>(positions),
               static_cast<const long long*>(slots), ldl, ldq, q_off, c_off, k_off, cq_off, Rq, heads, R, Rp, rotp, pairs, n_rows_form, eps, mscale};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = bf16 ? pdl::launch(k_latent_prep<__nv_bfloat16>, dim3(rows), dim3(256), 0, st, 1, p)
                       : pdl::launch(k_latent_prep<float>, dim3(rows), dim3(256), 0, st, 1, p);
  return e == cudaSuccess ? 0 : -1;
}

int tbv_op_latent_attn_rows(const void* qa, const void* cache, const void* tables, const void* seq_of_row, const void* ctx_lens,
                            const void* sink, void* out, int rows, int heads, int R, int Rp, int rotp, int block_size, int max_blocks,
                            int splits, float scale, int window, int bf16, void* stream) {
  if (R > Rp || (Rp % 16) || (rotp % 16) || window < 0) return -2;
  RowsParams p{qa, cache, static_cast<const int*>(tables), static_cast<const int*>(seq_of_row), static_cast<const int*>(ctx_lens),
               static_cast<const float*>(sink), out, heads, R, Rp, rotp, block_size, max_blocks, splits, 1, scale * kLog2e, scale, 0.f, nullptr, window, 0, nullptr, 0};
  return rows_form<kLatent>(p, rows, bf16, static_cast<cudaStream_t>(stream));
}

int tbv_op_latent_gather(const void* cache, const void* slots, void* c, void* kr, int n, int Rp, int rotp, void* stream) {
  if (n <= 0) return 0;
  if ((Rp % 16) || (rotp % 16)) return -2;
  cudaError_t e = pdl::launch(k_latent_gather, dim3((n + 7) / 8), dim3(256), 0, static_cast<cudaStream_t>(stream), 1,
                              static_cast<const uint4*>(cache), static_cast<const long long*>(slots), static_cast<uint4*>(c),
                              static_cast<uint4*>(kr), n, Rp / 8, rotp / 8);
  return e == cudaSuccess ? 0 : -1;
}

// 1 if the prefill form takes these sizes (bf16)
int tbv_op_latent_prefill_fits(int dimp, int rotp, int vdp) { return vdp <= 256 && prefill_smem(dimp + rotp, vdp) <= kMaxSmem ? 1 : 0; }

int tbv_op_latent_prefill(const void* q, const void* kv, const void* kr, const void* tiles, const void* sink, void* out, int ntiles,
                          int heads, int ldq, int q_rot_off, int ldkv, int v_off, int ldo, int dimp, int rotp, int vdp, float scale,
                          int window, void* stream) {
  if (ntiles <= 0) return 0;
  if ((dimp % 16) || (rotp % 16) || (vdp % 16) || (ldq % 8) || (ldkv % 8) || (q_rot_off % 8) || (v_off % 8) || ntiles > 65535 || window < 0) return -2;
  if (!tbv_op_latent_prefill_fits(dimp, rotp, vdp)) return -2;
  PrefillParams p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(kv), static_cast<const __nv_bfloat16*>(kr),
                  static_cast<__nv_bfloat16*>(out), static_cast<const int*>(tiles), static_cast<const float*>(sink),
                  ldq, q_rot_off, ldkv, v_off, ldo, dimp, rotp, vdp, scale * kLog2e, window};
  const size_t smem = prefill_smem(dimp + rotp, vdp);
  const dim3 grid(heads, ntiles);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (vdp <= 32) e = launch_prefill<2>(p, grid, smem, st);
  else if (vdp <= 64) e = launch_prefill<4>(p, grid, smem, st);
  else if (vdp <= 128) e = launch_prefill<8>(p, grid, smem, st);
  else e = launch_prefill<16>(p, grid, smem, st);
  if (e != cudaSuccess) fprintf(stderr, "[tbvops] latent prefill launch failed: %s\n", cudaGetErrorString(e));
  return e == cudaSuccess ? 0 : -1;
}

}  // extern "C"
