// delta_chunk.cu — the recurrence of delta.cu for many rows of a bf16 model, in chunks of 16 tokens on tensor cores.
//
// With P_t the product of the decays from the chunk's first token to t (per key channel), R_s the product after s to its last, and S the state before the chunk:
//   A_ts = sum_d q_t k_s (decays between s and t)  for s <= t,      B_ts the same with k_t for q_t, s < t
//   u = T (V - (k P) S)        T = (I + diag(beta) B)^-1 diag(beta)
//   o = (q P) S + A u          S <- diag(P_16) S + (k R)^T u
// Every factor is a running product of decays, at most 1: nothing is divided and no exponent can overflow, however strong the decay.  A and B are made of 4 x 4
// blocks: those on the diagonal from running products in registers; between neighbouring quarters of the chunk, and between its halves, as products of rows
// scaled to the boundary between them.  T: two 8 x 8 triangles by substitution, the block between them by two small products.
//
// S^T lives in the accumulators of the warps: warp w owns 16 value columns x all key channels.  As accumulator layout equals operand layout, S^T is also the left
// operand of both readouts, what they leave of V is that of the product with T, and u that of the last two.  v is bf16 as it stands.  All other operands are
// fp32 numbers carried as sums of kParts bf16 numbers, products of parts kept down to the kParts-th order (three parts: 24 bits, as fp32); what only enters the output,
// which is rounded to bf16 behind the head norm, in two.
//
// Eight warps of a CTA make the chunks' operands (they do not depend on the state), eight others take them through the products, one or two chunks behind; two sets
// of operands pass between them.  The two groups meet in named barriers only: `full` (operands of a set are there) and `empty` (its products are done).  If a
// CTA owns all value columns of its head, head norm, weight and gate follow here as well.
//
// With few sequences and heads most of the GPU would idle and every chunk would cost a maker's latency.  Then the two halves are kernels of their own: the sets
// of all chunks are made in parallel into memory (k_delta_make), and the products, their value columns shared out over several CTAs, find them there
// (k_delta_multiply: four warps fetch, four sets in flight).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <type_traits>

#include "../pdl.cuh"
#include "attn_mma.cuh"
#include "delta.cuh"
#include "ops.h"

using namespace attn_mma;
using delta_ops::Params;
using vec::f32x2;
using vec::mul2;
using vec::pack2;
using vec::unpack2;

namespace {

constexpr int kC = 16, kNW = 8, kNT = kNW * 32, kCols = kNW * 16;    // tokens of a chunk, warps and threads of a group, value columns of a CTA
constexpr int kParts = 3;
constexpr int kFetch = 128, kMakeChunks = 8;      // threads that fetch sets; chunks of a CTA that makes them

template <int DK>
struct Shape {
  static constexpr int kItems = DK / 16;                           // 16 channels x 16 tokens each; one per warp
  static constexpr int kPitch = DK * 2 + 16;                       // bytes; odd multiple of 16: ldmatrix without conflicts
  static constexpr int kVPitch = kCols * 2 + 16;
  static constexpr int kAPitch = kC * 2 + 16;
  static constexpr int kOPitch = kCols + 4;                        // floats
  // a set of operands, byte offsets in it
  static constexpr int oQ = 0;                                     // q P                 [2][16][pitch]
  static constexpr int oK = oQ + 2 * kC * kPitch;                  // k P                 [parts][16][pitch]
  static constexpr int oR = oK + kParts * kC * kPitch;             // k R                 [parts][16][pitch]
  static constexpr int oA = oR + kParts * kC * kPitch;             // A                   [2][16][apitch]
  static constexpr int oT = oA + 2 * kC * kAPitch;                 // T                   [parts][16][apitch]
  static constexpr int oE = oT + kParts * kC * kAPitch;            // P_16                [DK] fp32
  static constexpr int kStored = oE + DK * 4;                      // what a set in memory holds
  static constexpr int oV = kStored;                               // v                   [16][vpitch]
  static constexpr int oL = oV + kC * kVPitch;                     // diag(beta) B        [16][17] fp32
  static constexpr int oB = oL + 16 * 17 * 4;                      // step sizes          [16] fp32
  static constexpr int kSet = oB + kC * 4;
  static_assert(kStored % 16 == 0 && kSet % 16 == 0, "16-byte copies");
};
// Dynamic shared memory of a CTA that makes operands: its sets, then what the makers have for themselves.
template <int DK, int SETS, int RAWS>
struct Layout : Shape<DK> {
  using B = Shape<DK>;
  using B::kItems;
  using B::kPitch;
  static constexpr int oTa = SETS * B::kSet;                            // blocks: left rows   [parts][2 kinds][16][pitch]  (8 of q, 8 of k)
  static constexpr int oTb = oTa + kParts * 32 * kPitch;           //         right rows  [parts][2 kinds][8][pitch]
  static constexpr int oZ = oTb + kParts * 16 * kPitch;            // raw decay inputs [16][DK] fp32, q and k [16][DK] bf16 each; RAWS chunks
  static constexpr int kRq = kC * DK * 4, kRk = kRq + kC * DK * 2, kRaw = kRk + kC * DK * 2;
  static constexpr int oF = oZ + RAWS * kRaw;                         // factors of q, of k, step sizes [2 chunks][3][16] fp32
  static constexpr int oTri = oF + 6 * kC * 4;                     // diagonal blocks     [items][4 quarters][16] fp32
  static constexpr int oOff = oTri + (kItems + 1) * 256;           // the other blocks' sums [warps][2][16][8] fp32
  static constexpr int oI = oOff + kNW * 1024;                     // I + diag(beta) B inverted [16][17] fp32, a product [8][17]
  static constexpr int oO = oI + 24 * 17 * 4;                      // o                   [16][opitch] fp32 (both halves in one kernel)
  static constexpr int kBytes = oO + (SETS == 2 ? kC * B::kOPitch * 4 : 0);
  static_assert(oTa % 16 == 0 && oZ % 16 == 0 && oF % 16 == 0 && oO % 16 == 0 && kBytes <= (SETS == 2 ? int(kMaxSmem) : 113 * 1024), "shared memory; two CTAs per SM");
};
template <int DK> using Both = Layout<DK, 2, 2>;
template <int DK> using Make = Layout<DK, 1, 1>;

// Named barriers (0 is __syncthreads): one inside each group, `full` and `empty` of up to four sets of operands.
enum Bar : int { kMakers = 1, kProducts = 2, kFull = 3, kEmpty = 7 };
__device__ __forceinline__ void bar_sync(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
__device__ __forceinline__ void bar_arrive(int id, int threads) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

__device__ __forceinline__ void st_shared(uint32_t addr, uint32_t v) { asm volatile("st.shared.b32 [%0], %1;" ::"r"(addr), "r"(v) : "memory"); }
__device__ __forceinline__ float2 of2(f32x2 v) {
  float2 r;
  unpack2(v, r.x, r.y);
  return r;
}
// (x, y) as sums of N bf16 pairs: all but the last are cut off behind eight bits, so that what is left is exact
template <int N>
__device__ __forceinline__ void split(float x, float y, uint32_t* part) {
#pragma unroll
  for (int i = 0; i + 1 < N; i++) {
    const uint32_t u = __float_as_uint(x), v = __float_as_uint(y);
    part[i] = __byte_perm(u, v, 0x7632);
    x -= __uint_as_float(u & 0xffff0000u);
    y -= __uint_as_float(v & 0xffff0000u);
  }
  part[N - 1] = pack_bf16(x, y);
}
// two neighbouring channels to `addr`, their parts `stride` bytes apart
template <int N>
__device__ __forceinline__ void put(f32x2 v, uint32_t addr, uint32_t stride) {
  uint32_t part[N];
  const float2 f = of2(v);
  split<N>(f.x, f.y, part);
#pragma unroll
  for (int i = 0; i < N; i++) st_shared(addr + i * stride, part[i]);
}
// accumulators [2 tiles of 8 columns][4] as a left operand of 16 columns
template <int N>
__device__ __forceinline__ void as_left(const float (*v)[4], uint32_t (*a)[4]) {
#pragma unroll
  for (int j = 0; j < 4; j++) {
    uint32_t part[N];
    split<N>(v[j >> 1][(j & 1) * 2], v[j >> 1][(j & 1) * 2 + 1], part);
#pragma unroll
    for (int i = 0; i < N; i++) a[i][j] = part[i];
  }
}

struct Job {                        // what one CTA works on, and where a thread stands in its group
  int h, g, first, n, nc, slot, vb, cols;  // vb: first of its value columns
  int tid, warp, lane, row16, l16;  // 16 lanes per row of a chunk
};
__device__ __forceinline__ Job job_of(const Params& p, const int* group, int h, int vb, int cols, int tid) {
  Job w;
  w.h = h;
  w.g = h / (p.heads / p.kv_heads);
  w.first = group[0];
  w.n = group[1];
  w.slot = group[2];
  w.nc = (w.n + kC - 1) / kC;
  w.vb = vb;
  w.cols = cols;
  w.tid = tid;
  w.warp = tid >> 5;
  w.lane = tid & 31;
  w.row16 = tid >> 4;
  w.l16 = tid & 15;
  return w;
}
// Sets in memory: that of chunk c of group gi, head h is number (first / 16 + gi + c) * heads + h (different for all chunks of a batch).
__device__ __forceinline__ int first_set(const Job& w, int gi) { return w.first / kC + gi; }

// ---- the makers -----------------------------------------------------------------------------------------------------------
// Chunks c0 .. c1 - 1.  sets null: they go to the products of this CTA; otherwise to memory, chunk c to sets + c * stride.
template <int DK, bool STORE>
__device__ __forceinline__ void make_operands(const Params& p, uint8_t* sm, const Job& w, int c0, int c1, uint8_t* sets, size_t stride) {
  using S = typename std::conditional<STORE, Make<DK>, Both<DK>>::type;
  constexpr int kRaws = STORE ? 0 : 1;          // mask of the raw buffers
  const int tid = w.tid, warp = w.warp, lane = w.lane, r8 = lane >> 2, quad = lane & 3, row16 = w.row16, l16 = w.l16, n = w.n;
  const uint32_t base = smem_addr(sm);
  const float rate2 = -p.rate[w.h] * kLog2e, qscale = rsqrtf(float(p.dim));
  const __nv_bfloat16* qg = static_cast<const __nv_bfloat16*>(p.q) + size_t(w.g) * p.Dp;
  const __nv_bfloat16* kg = static_cast<const __nv_bfloat16*>(p.k) + size_t(w.g) * p.Dp;
  const __nv_bfloat16* vg = static_cast<const __nv_bfloat16*>(p.v) + size_t(w.h) * p.Vp + w.vb;
  const float* zg = p.z + size_t(w.h) * p.Dp;

  // rows of chunk c on their way to shared memory; missing rows are zeros: they decay nothing, write nothing and read nothing
  auto issue = [&](int c) {
    const size_t r = size_t(w.first + c * kC + row16);
    const uint32_t raw = base + S::oZ + (c & kRaws) * S::kRaw;
    if (c * kC + row16 >= n) {
      for (int x = l16; x < DK / 4; x += 16) st_zero16(raw + (row16 * DK + x * 4) * 4);
      for (int x = l16; x < DK / 4; x += 16) st_zero16(raw + S::kRq + (x >= DK / 8 ? S::kRk - S::kRq : 0) + (row16 * DK + x % (DK / 8) * 8) * 2);
      return;
    }
    for (int x = l16; x < p.Dp / 4; x += 16) cp_async16(raw + (row16 * DK + x * 4) * 4, zg + r * p.ldz + x * 4);
    for (int x = l16; x < p.Dp / 8; x += 16) {
      cp_async16(raw + S::kRq + (row16 * DK + x * 8) * 2, qg + r * p.ld + x * 8);
      cp_async16(raw + S::kRk + (row16 * DK + x * 8) * 2, kg + r * p.ld + x * 8);
    }
  };
  auto issue_v = [&](int c, uint32_t set) {                         // missing rows are zeros
    const uint32_t dst = set + S::oV + row16 * S::kVPitch + l16 * 16;
    if (l16 >= min(w.cols, p.Vp - w.vb) / 8) return;
    if (c * kC + row16 < n) cp_async16(dst, vg + size_t(w.first + c * kC + row16) * p.ld + l16 * 8);
    else st_zero16(dst);
  };
  __nv_bfloat16 beta_next = __float2bfloat16_rn(0.f);               // step size of row `tid` of the chunk on its way
  auto fetch_beta = [&](int c) {
    if (tid < kC && c * kC + tid < n) beta_next = static_cast<const __nv_bfloat16*>(p.beta)[size_t(w.first + c * kC + tid) * p.ldx + w.h];
  };
  // factors that make rows of q and k unit vectors (of rows that this thread's own copies brought), step sizes
  auto factors_of = [&](int c) { return reinterpret_cast<float*>(sm + S::oF) + (c & 1) * 3 * kC; };
  auto norms = [&](int c) {
    const uint8_t* raw = sm + S::oZ + (c & kRaws) * S::kRaw;
    float *factors = factors_of(c), sq = 0.f, sk = 0.f;
    for (int x = l16; x < p.Dp / 8; x += 16) {
      float f[8], k[8];
      vec::load8(reinterpret_cast<const __nv_bfloat16*>(raw + S::kRq) + row16 * DK + x * 8, f);
      vec::load8(reinterpret_cast<const __nv_bfloat16*>(raw + S::kRk) + row16 * DK + x * 8, k);
#pragma unroll
      for (int e = 0; e < 8; e++) { sq = fmaf(f[e], f[e], sq); sk = fmaf(k[e], k[e], sk); }
    }
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) {
      sq += __shfl_xor_sync(0xffffffffu, sq, o);
      sk += __shfl_xor_sync(0xffffffffu, sk, o);
    }
    if (l16 == 0) {
      factors[row16] = qscale / sqrtf(sq + delta_ops::kUnitEps);
      factors[kC + row16] = 1.0f / sqrtf(sk + delta_ops::kUnitEps);
    }
    if (tid < kC) factors[2 * kC + tid] = vec::sigmoid<__nv_bfloat16>(__bfloat162float(beta_next));
  };
  // Operands of chunk c, a warp takes 16 channels, a lane two of them over four tokens (a quarter of the chunk).  First what the scores of a chunk are made of;
  // the operands of the state's products, which need their set free, are left in registers: q and k times the decays from their quarter's start (their own
  // included), k times those behind it in its quarter, products of the decays over the quarters before and after.
  f32x2 qr[4], kr[4], kc[4], before = 0ull, after = 0ull, all = 0ull;
  const int quarter = lane >> 3, d = warp * 16 + (lane & 7) * 2;
  const bool odd = quarter & 1, late = quarter & 2, item = warp * 16 < p.Dp;
  auto scores = [&](int c) {
    if (!item) return;
    const uint8_t* raw = sm + S::oZ + (c & kRaws) * S::kRaw;
    const float* factors = factors_of(c);
    f32x2 a[4], q[4], k[4];
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int t = quarter * 4 + j;
      const float2 z = *reinterpret_cast<const float2*>(raw + (t * DK + d) * 4);
      const uint32_t qb = *reinterpret_cast<const uint32_t*>(raw + S::kRq + (t * DK + d) * 2), kb = *reinterpret_cast<const uint32_t*>(raw + S::kRk + (t * DK + d) * 2);
      const float fq = factors[t], fk = factors[kC + t];
      const float a0 = vec::pow2<__nv_bfloat16>(z.x * rate2), a1 = vec::pow2<__nv_bfloat16>(z.y * rate2);
      a[j] = pack2(a0, a1);
      q[j] = mul2(pack2(__uint_as_float(qb << 16), __uint_as_float(qb & 0xffff0000u)), pack2(fq, fq));
      k[j] = mul2(pack2(__uint_as_float(kb << 16), __uint_as_float(kb & 0xffff0000u)), pack2(fk, fk));
    }
    // products over quarters: t1 of quarter ^ 1, t23 of the two others
    const f32x2 tot = mul2(mul2(a[0], a[1]), mul2(a[2], a[3]));
    const f32x2 t1 = __shfl_xor_sync(0xffffffffu, tot, 8), both = mul2(tot, t1), t23 = __shfl_xor_sync(0xffffffffu, both, 16), one = pack2(1.f, 1.f);
    before = mul2(odd ? t1 : one, late ? t23 : one);
    after = mul2(odd ? one : t1, late ? one : t23);
    all = mul2(both, t23);
    const f32x2 half = odd == late ? t1 : one;                      // to (quarters 0, 1) and from (2, 3) the middle of the chunk: over quarter 1, over quarter 2
    constexpr uint32_t ka = 32 * S::kPitch, kb = 16 * S::kPitch;
    const uint32_t col = base + d * 2;
    f32x2 run = one;
#pragma unroll
    for (int j = 3; j >= 0; j--) {
      kc[j] = mul2(k[j], run);
      run = mul2(run, a[j]);
    }
    run = one;
    const uint32_t ta = col + S::oTa + (late ? 4 : 0) * S::kPitch, tb = col + S::oTb + (late ? 4 : 0) * S::kPitch;
    const uint32_t ua = col + S::oTa + (16 + (odd ? 4 : 0)) * S::kPitch, ub = col + S::oTb + (8 + (odd ? 4 : 0)) * S::kPitch;
#pragma unroll
    for (int j = 0; j < 4; j++) {
      run = mul2(run, a[j]);
      qr[j] = mul2(q[j], run);
      kr[j] = mul2(k[j], run);
      // between neighbouring quarters: rows of quarters 1 and 3 against those of 0 and 2
      put<kParts>(odd ? qr[j] : kc[j], (odd ? ta : tb) + j * S::kPitch, odd ? ka : kb);
      if (odd) put<kParts>(kr[j], ta + (8 + j) * S::kPitch, ka);
      // between the halves
      put<kParts>(mul2(late ? qr[j] : kc[j], half), (late ? ua : ub) + j * S::kPitch, late ? ka : kb);
      if (late) put<kParts>(mul2(kr[j], half), ua + (8 + j) * S::kPitch, ka);
    }
    // the diagonal block of this quarter: (t, s <= t) for q, then (t, s < t) for k, summed over the 8 lanes that share it
    float val[16];
#pragma unroll
    for (int t = 0; t < 4; t++) {
#pragma unroll
      for (int s = 0; s < t; s++) k[s] = mul2(k[s], a[t]);          // k_s times the decays between s and t
#pragma unroll
      for (int s = 0; s <= t; s++) {
        const float2 v = of2(mul2(q[t], k[s]));
        val[t * (t + 1) / 2 + s] = v.x + v.y;
        if (s < t) {
          const float2 x = of2(mul2(k[t], k[s]));
          val[10 + t * (t - 1) / 2 + s] = x.x + x.y;
        }
      }
    }
    int idx = 0;
#pragma unroll
    for (int c = 8; c >= 2; c >>= 1) {
      const int off = c / 2;
      const bool up = lane & off;
#pragma unroll
      for (int j = 0; j < 8; j++)
        if (j < c) {
          const float send = up ? val[j] : val[j + c], keep = up ? val[j + c] : val[j];
          val[j] = keep + __shfl_xor_sync(0xffffffffu, send, off);
        }
      idx += up ? c : 0;
    }
    *reinterpret_cast<float2*>(sm + S::oTri + ((warp * 4 + quarter) * 16 + idx) * 4) = make_float2(val[0], val[1]);
  };
  auto operands = [&](uint32_t set, uint8_t* set_p) {
    if (!item) return;
    constexpr uint32_t kp = kC * S::kPitch;
    const uint32_t own = set + quarter * 4 * S::kPitch + d * 2;
    if (quarter == 0) *reinterpret_cast<float2*>(set_p + S::oE + d * 4) = of2(all);
#pragma unroll
    for (int j = 0; j < 4; j++) {
      put<2>(mul2(qr[j], before), own + S::oQ + j * S::kPitch, kp);
      put<kParts>(mul2(kr[j], before), own + S::oK + j * S::kPitch, kp);
      put<kParts>(mul2(kc[j], after), own + S::oR + j * S::kPitch, kp);
    }
  };
  // the blocks between quarters and halves: left rows against right rows, k steps shared out over the warps
  auto blocks = [&]() {
    if (!item) return;
    float acc[2][4] = {};
    uint32_t a[2][kParts][4], b[2][kParts][2];
#pragma unroll
    for (int kind = 0; kind < 2; kind++)
#pragma unroll
      for (int i = 0; i < kParts; i++) {
        ldmatrix_x4(base + S::oTa + (i * 32 + kind * 16 + (lane & 15)) * S::kPitch + warp * 32 + (lane >> 4) * 16, a[kind][i]);
        ldmatrix_x2(base + S::oTb + (i * 16 + kind * 8 + (lane & 7)) * S::kPitch + warp * 32 + ((lane >> 3) & 1) * 16, b[kind][i]);
      }
#pragma unroll
    for (int i = kParts - 1; i >= 0; i--)
#pragma unroll
      for (int j = kParts - 1 - i; j >= 0; j--)
#pragma unroll
        for (int kind = 0; kind < 2; kind++) mma_bf16(acc[kind], a[kind][i], b[kind][j][0], b[kind][j][1]);
#pragma unroll
    for (int kind = 0; kind < 2; kind++) {
      float* off = reinterpret_cast<float*>(sm + S::oOff) + (warp * 2 + kind) * 128;
      *reinterpret_cast<float2*>(off + r8 * 8 + quad * 2) = make_float2(acc[kind][0], acc[kind][1]);
      *reinterpret_cast<float2*>(off + (r8 + 8) * 8 + quad * 2) = make_float2(acc[kind][2], acc[kind][3]);
    }
  };
  // A and diag(beta) B from their pieces, an element per thread
  auto assemble = [&](uint8_t* set_p, const float* factors) {
    const int t = tid >> 4, s = tid & 15, qt = t >> 2, qs = s >> 2, items = p.Dp / 16;
    float vq = 0.f, vk = 0.f;
    if (s <= t) {
      const float *at, *ak;
      int step;
      if (qt == qs) {
        const int tt = t & 3, ss = s & 3;
        at = reinterpret_cast<const float*>(sm + S::oTri) + qt * 16 + tt * (tt + 1) / 2 + ss;
        ak = reinterpret_cast<const float*>(sm + S::oTri) + qt * 16 + 10 + tt * (tt - 1) / 2 + ss;     // (s = t: not used)
        step = 64;
      } else {
        const bool far = (qt ^ qs) & 2;
        at = reinterpret_cast<const float*>(sm + S::oOff) + (far ? 128 + (t - 8) * 8 + s : ((qt >> 1) * 4 + (t & 3)) * 8 + (qs >> 1) * 4 + (s & 3));
        ak = at + 64;
        step = 256;
      }
#pragma unroll
      for (int i = 0; i < S::kItems; i++)
        if (i < items) { vq += at[i * step]; vk += ak[i * step]; }
    }
    const __nv_bfloat16 hi = __float2bfloat16_rn(vq);
    reinterpret_cast<__nv_bfloat16*>(set_p + S::oA + t * S::kAPitch)[s] = hi;
    reinterpret_cast<__nv_bfloat16*>(set_p + S::oA + (kC + t) * S::kAPitch)[s] = __float2bfloat16_rn(vq - __bfloat162float(hi));
    reinterpret_cast<float*>(set_p + S::oL)[t * 17 + s] = s < t ? vk * factors[2 * kC + t] : 0.f;
    if (tid < kC) reinterpret_cast<float*>(set_p + S::oB)[tid] = factors[2 * kC + tid];
  };
  // T, by one warp
  auto invert = [&](uint32_t set, const uint8_t* set_p) {
    const float *L = reinterpret_cast<const float*>(set_p + S::oL), *beta = reinterpret_cast<const float*>(set_p + S::oB);
    float *I = reinterpret_cast<float*>(sm + S::oI), *M = I + 16 * 17;
    const int b8 = lane & 8, j = lane & 7;                          // lanes 16 .. 31 repeat the others
    float x[8];
#pragma unroll
    for (int t = 0; t < 8; t++) {
      float v = t == j ? 1.f : 0.f;
#pragma unroll
      for (int s = 0; s < t; s++) v = fmaf(-L[(b8 + t) * 17 + b8 + s], x[s], v);
      x[t] = v;
    }
    if (lane < 16) {
#pragma unroll
      for (int t = 0; t < 8; t++) I[(b8 + t) * 17 + b8 + j] = x[t];
    }
    __syncwarp();
    const int c = quad * 2;
    float m0 = 0.f, m1 = 0.f;
#pragma unroll
    for (int s = 0; s < 8; s++) {
      const float l = L[(8 + r8) * 17 + s];
      m0 = fmaf(l, I[s * 17 + c], m0);
      m1 = fmaf(l, I[s * 17 + c + 1], m1);
    }
    M[r8 * 17 + c] = m0;
    M[r8 * 17 + c + 1] = m1;
    __syncwarp();
    m0 = m1 = 0.f;
#pragma unroll
    for (int s = 0; s < 8; s++) {
      const float l = I[(8 + r8) * 17 + 8 + s];
      m0 = fmaf(-l, M[s * 17 + c], m0);
      m1 = fmaf(-l, M[s * 17 + c + 1], m1);
    }
    // rows r8 and 8 + r8, columns c, c + 1 of both halves
    auto out = [&](int t, int s, float v0, float v1) {
      uint32_t part[kParts];
      split<kParts>(v0 * beta[s], v1 * beta[s + 1], part);
#pragma unroll
      for (int i = 0; i < kParts; i++) st_shared(set + S::oT + (i * kC + t) * S::kAPitch + s * 2, part[i]);
    };
    out(r8, c, I[r8 * 17 + c], I[r8 * 17 + c + 1]);
    out(r8, 8 + c, 0.f, 0.f);
    out(8 + r8, c, m0, m1);
    out(8 + r8, 8 + c, I[(8 + r8) * 17 + 8 + c], I[(8 + r8) * 17 + 8 + c + 1]);
  };
  issue(c0);
  cp_async_commit();
  fetch_beta(c0);
  for (int i = tid; i < S::oZ / 16; i += kNT) st_zero16(base + i * 16);     // operand rows of channels beyond Dp stay zero
  cp_async_wait<0>();
  norms(c0);
  bar_sync(kMakers, kNT);
  for (int c = c0; c < c1; c++) {                                   // the raw rows of chunk c are there, and their factors
    const int b = STORE ? 0 : c & 1;
    uint8_t* set_p = sm + b * S::kSet;
    const uint32_t set = base + b * S::kSet;
    auto next = [&]() {
      if (c + 1 < c1) {
        issue(c + 1);
        fetch_beta(c + 1);
      }
      cp_async_commit();
    };
    if (!STORE) next();
    scores(c);
    bar_sync(kMakers, kNT);
    if (STORE) next();                                              // into the rows just read
    if (!STORE) {
      if (c >= 2) bar_sync(kEmpty + b, 2 * kNT);                    // the products of chunk c - 2 are done
      issue_v(c, set);
      cp_async_commit();
    }
    blocks();
    operands(set, set_p);
    bar_sync(kMakers, kNT);
    assemble(set_p, factors_of(c));
    if (c + 1 < c1) {
      cp_async_wait<STORE ? 0 : 1>();
      norms(c + 1);
    }
    bar_sync(kMakers, kNT);
    if (warp == 0) invert(set, set_p);
    if (STORE) {
      bar_sync(kMakers, kNT);
      uint4* to = reinterpret_cast<uint4*>(sets + c * stride);
      for (int i = tid; i < S::kStored / 16; i += kNT) to[i] = reinterpret_cast<const uint4*>(set_p)[i];
    } else {
      cp_async_wait<0>();                                           // v
      bar_arrive(kFull + b, 2 * kNT);
    }
  }
  cp_async_wait<0>();
}

// ---- the products -----------------------------------------------------------------------------------------------------------
// SETS 2: beside the makers, o of a chunk stays here for its norm if p.o is null.  SETS 4: beside the warps that fetch.
// DS warps share the 16 value columns of a warp: each has DK / DS of the channels, their readouts are summed through shared memory (at `xch`).
template <int DK, int SETS, int DS>
__device__ __forceinline__ void multiply(const Params& p, uint8_t* sm, const Job& w, float* xch) {
  using S = Both<DK>;
  constexpr int kMeet = SETS == 2 ? 2 * kNT : kNT + kFetch;        // threads that meet in a barrier of a set
  const int lane = w.lane, r8 = lane >> 2, quad = lane & 3, row16 = w.row16, l16 = w.l16, n = w.n;
  const uint32_t base = smem_addr(sm);
  const bool fresh = p.positions[w.first] == 0, fused = SETS == 2 && p.o == nullptr;
  constexpr int DW = DK / DS;
  const int part = w.warp % DS, own = w.warp / DS, d0 = part * DW;  // channels from d0 on
  const int v0 = w.vb + own * 16;                                   // first value column of the warp
  const bool mma_warp = own * 16 < w.cols && v0 < p.Vp;
  float st[DW / 8][4];      // S^T: value column v0 + r8 (+ 8), channels d0 + 8 i + 2 quad (+ 1)
  float* state = p.state + (size_t(w.slot) * p.heads + w.h) * p.Dp * p.Vp;
#pragma unroll
  for (int i = 0; i < DW / 8; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int d = d0 + i * 8 + quad * 2 + (j & 1), v = v0 + r8 + (j >> 1) * 8;
      st[i][j] = !mma_warp || fresh || d >= p.Dp ? 0.f : state[size_t(d) * p.Vp + v];
    }
  const uint32_t brow = (lane & 7) + ((lane >> 4) << 3), bcol = ((lane >> 3) & 1) * 16;    // right operands stored [n][k]
  for (int c = 0; c < w.nc; c++) {
    const int b = c % SETS, at = c * kC;
    const uint32_t set = base + b * S::kSet;
    vec::Raw8<__nv_bfloat16> gate;
    if (fused && at + row16 < n && l16 * 8 < p.Vp)
      gate.load(static_cast<const __nv_bfloat16*>(p.gate) + size_t(w.first + at + row16) * p.ldg + size_t(w.h) * p.Vp + l16 * 8);
    bar_sync(kFull + b, kMeet);
    float o[2][2][4] = {}, x[2][2][4] = {};
    if (mma_warp) {
      // (q P) S and (k P) S, two sums each for even and odd k steps: value column as above, tokens 8 i + 2 quad (+ 1)
#pragma unroll
      for (int ks = 0; ks < DW / 16; ks += 2) {
        uint32_t s[2][kParts][4], r[2][4];
        as_left<kParts>(st + 2 * ks, s[0]);
        as_left<kParts>(st + 2 * ks + 2, s[1]);
#pragma unroll
        for (int j = kParts - 1; j >= 0; j--) {
#pragma unroll
          for (int e = 0; e < 2; e++) ldmatrix_x4(set + S::oK + (j * kC + brow) * S::kPitch + bcol + d0 * 2 + (ks + e) * 32, r[e]);
#pragma unroll
          for (int i = kParts - 1 - j; i >= 0; i--)
#pragma unroll
            for (int e = 0; e < 2; e++) {
              mma_bf16(x[e][0], s[e][i], r[e][0], r[e][1]);
              mma_bf16(x[e][1], s[e][i], r[e][2], r[e][3]);
            }
        }
#pragma unroll
        for (int j = 1; j >= 0; j--) {
#pragma unroll
          for (int e = 0; e < 2; e++) ldmatrix_x4(set + S::oQ + (j * kC + brow) * S::kPitch + bcol + d0 * 2 + (ks + e) * 32, r[e]);
#pragma unroll
          for (int i = 1 - j; i >= 0; i--)
#pragma unroll
            for (int e = 0; e < 2; e++) {
              mma_bf16(o[e][0], s[e][i], r[e][0], r[e][1]);
              mma_bf16(o[e][1], s[e][i], r[e][2], r[e][3]);
            }
        }
      }
#pragma unroll
      for (int i = 0; i < 2; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) { x[0][i][j] += x[1][i][j]; o[0][i][j] += o[1][i][j]; }
      if constexpr (DS > 1) {
        float* mine = xch + w.warp * 512 + lane;
#pragma unroll
        for (int i = 0; i < 16; i++) mine[i * 32] = i < 8 ? x[0][i >> 2][i & 3] : o[0][(i >> 2) & 1][i & 3];
      }
    }
    if constexpr (DS > 1) bar_sync(kProducts, kNT);
    if (mma_warp) {
      if constexpr (DS > 1) {                   // in the same order in all of them
        float sum[16];
#pragma unroll
        for (int i = 0; i < 16; i++) {
          sum[i] = 0.f;
#pragma unroll
          for (int k = 0; k < DS; k++) sum[i] += xch[(own * DS + k) * 512 + i * 32 + lane];
          if (i < 8) x[0][i >> 2][i & 3] = sum[i];
          else o[0][(i >> 2) & 1][i & 3] = sum[i];
        }
      }
      uint32_t l[kParts][4], f[4];
      ldmatrix_x4_trans(set + S::oV + brow * S::kVPitch + own * 32 + bcol, f);      // v^T: stored [token][column]
#pragma unroll
      for (int j = 0; j < 4; j++) {
        float* y = &x[0][j >> 1][(j & 1) * 2];
        y[0] = __uint_as_float(f[j] << 16) - y[0];
        y[1] = __uint_as_float(f[j] & 0xffff0000u) - y[1];
      }
      float u[2][4] = {};
      as_left<kParts>(x[0], l);
#pragma unroll
      for (int j = kParts - 1; j >= 0; j--) {
        ldmatrix_x4(set + S::oT + (j * kC + brow) * S::kAPitch + bcol, f);
#pragma unroll
        for (int i = kParts - 1 - j; i >= 0; i--) {
          mma_bf16(u[0], l[i], f[0], f[1]);
          mma_bf16(u[1], l[i], f[2], f[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < DW / 8; i++) {
        const float2 e = *reinterpret_cast<const float2*>(sm + b * S::kSet + S::oE + (d0 + i * 8 + quad * 2) * 4);
        st[i][0] *= e.x; st[i][1] *= e.y; st[i][2] *= e.x; st[i][3] *= e.y;
      }
      as_left<kParts>(u, l);
      if (part == 0) {
        float q[2][4] = {};
#pragma unroll
        for (int j = 1; j >= 0; j--) {
          ldmatrix_x4(set + S::oA + (j * kC + brow) * S::kAPitch + bcol, f);
#pragma unroll
          for (int i = 1 - j; i >= 0; i--) {
            mma_bf16(i ? q[0] : o[0][0], l[i], f[0], f[1]);
            mma_bf16(i ? q[1] : o[0][1], l[i], f[2], f[3]);
          }
        }
#pragma unroll
        for (int i = 0; i < 2; i++)
#pragma unroll
          for (int j = 0; j < 4; j++) o[0][i][j] += q[i][j];
      }
#pragma unroll
      for (int i = 0; i < DW / 16; i += 2)
#pragma unroll
        for (int j = kParts - 1; j >= 0; j--) {                     // smallest part first
          uint32_t r[2][4];
#pragma unroll
          for (int e = 0; e < 2; e++) ldmatrix_x4_trans(set + S::oR + (j * kC + (lane & 15)) * S::kPitch + d0 * 2 + (i + e) * 32 + (lane >> 4) * 16, r[e]);
#pragma unroll
          for (int y = kParts - 1 - j; y >= 0; y--)
#pragma unroll
            for (int e = 0; e < 2; e++) {
              mma_bf16(st[2 * (i + e)], l[y], r[e][0], r[e][1]);
              mma_bf16(st[2 * (i + e) + 1], l[y], r[e][2], r[e][3]);
            }
        }
#pragma unroll
      for (int i = 0; i < 2; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
          const int t = i * 8 + quad * 2 + (j & 1), v = r8 + (j >> 1) * 8;
          const float y = o[0][i][j];
          if (part != 0) continue;
          if (fused) reinterpret_cast<float*>(sm + S::oO)[t * S::kOPitch + own * 16 + v] = y;
          else if (at + t < n) p.o[(size_t(w.first + at + t) * p.heads + w.h) * p.Vp + v0 + v] = y;
        }
    }
    if (c + SETS < w.nc) bar_arrive(kEmpty + b, kMeet);
    if (!fused) continue;
    // head norm, weight and gate; a row per 16 lanes, 8 columns per lane.  (The next chunk's o is written behind its `full`, which waits for all of these warps.)
    bar_sync(kProducts, kNT);
    const int v = l16 * 8;
    float y[8], ss = 0.f;
    vec::load8(reinterpret_cast<const float*>(sm + S::oO) + row16 * S::kOPitch + v, y);
    if (v >= p.Vp) {
#pragma unroll
      for (int e = 0; e < 8; e++) y[e] = 0.f;
    }
#pragma unroll
    for (int e = 0; e < 8; e++) ss = fmaf(y[e], y[e], ss);
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (at + row16 < n && v < p.Vp) {
      const float r = 1.0f / sqrtf(ss / float(p.vdim) + p.eps);
      float gt[8], wt[8];
      gate.unpack(gt);
      vec::load8(p.norm + v, wt);
#pragma unroll
      for (int e = 0; e < 8; e++) y[e] = y[e] * r * wt[e] * vec::sigmoid<__nv_bfloat16>(gt[e]);
      vec::store8(static_cast<__nv_bfloat16*>(p.out) + size_t(w.first + at + row16) * p.ldo + size_t(w.h) * p.Vp + v, y);
    }
  }
  if (mma_warp) {
#pragma unroll
    for (int i = 0; i < DW / 8; i++)
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const int d = d0 + i * 8 + quad * 2 + (j & 1), v = v0 + r8 + (j >> 1) * 8;
        if (d < p.Dp) state[size_t(d) * p.Vp + v] = st[i][j];
      }
  }
}

// Four warps that bring sets from memory, and the values of their columns, three chunks ahead.
template <int DK>
__device__ __forceinline__ void fetch_operands(const Params& p, uint8_t* sm, const Job& w, const uint8_t* sets, size_t stride) {
  using S = Shape<DK>;
  const uint32_t base = smem_addr(sm);
  const int units = min(w.cols, p.Vp - w.vb) / 8;
  const __nv_bfloat16* vg = static_cast<const __nv_bfloat16*>(p.v) + size_t(w.h) * p.Vp + w.vb;
  auto issue = [&](int c) {
    if (c < w.nc) {
      const uint32_t set = base + (c & 3) * S::kSet;
      const uint8_t* from = sets + c * stride;
      for (int i = w.tid; i < S::kStored / 16; i += kFetch) cp_async16(set + i * 16, from + i * 16);
      for (int i = w.tid; i < kC * units; i += kFetch) {            // missing rows are zeros
        const int t = i / units, x = i - t * units;
        const uint32_t dst = set + S::oV + t * S::kVPitch + x * 16;
        if (c * kC + t < w.n) cp_async16(dst, vg + size_t(w.first + c * kC + t) * p.ld + x * 8);
        else st_zero16(dst);
      }
    }
    cp_async_commit();
  };
  for (int c = 0; c < 3; c++) issue(c);
  for (int c = 0; c < w.nc; c++) {
    cp_async_wait<2>();                                             // chunk c
    bar_arrive(kFull + (c & 3), kNT + kFetch);
    if (c >= 1 && c + 3 < w.nc) bar_sync(kEmpty + ((c + 3) & 3), kNT + kFetch);   // the products of chunk c - 1 are done
    issue(c + 3);
  }
  cp_async_wait<0>();
}

// registers of the launch, 128 per thread, shared out anew
template <int N> __device__ __forceinline__ void more_registers() { asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(N)); }
template <int N> __device__ __forceinline__ void fewer_registers() { asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(N)); }

template <int DK>
__global__ void __launch_bounds__(2 * kNT, 1) k_delta_chunk(const Params p, const int* groups) {
  extern __shared__ __align__(16) uint8_t sm[];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const Job w = job_of(p, groups + 4 * blockIdx.x, blockIdx.y, blockIdx.z * kCols, kCols, threadIdx.x % kNT);
  if (threadIdx.x < kNT) {
    more_registers<152>();
    multiply<DK, 2, 1>(p, sm, w, nullptr);
  } else {
    fewer_registers<104>();
    make_operands<DK, false>(p, sm, w, 0, w.nc, nullptr, 0);
  }
}

// CTA (x, head): the sets numbered x * kMakeChunks .. of all groups
template <int DK>
__global__ void __launch_bounds__(kNT, 2) k_delta_make(const Params p, const int* groups, int ngroups, uint8_t* sets) {
  extern __shared__ __align__(16) uint8_t sm[];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const size_t stride = size_t(p.heads) * Shape<DK>::kStored;
  for (int gi = 0; gi < ngroups; gi++) {
    const Job w = job_of(p, groups + 4 * gi, blockIdx.y, 0, kCols, threadIdx.x);
    const int s0 = first_set(w, gi), c0 = max(0, int(blockIdx.x) * kMakeChunks - s0), c1 = min(w.nc, int(blockIdx.x + 1) * kMakeChunks - s0);
    if (c0 < c1) {
      make_operands<DK, true>(p, sm, w, c0, c1, sets + s0 * stride + size_t(w.h) * Shape<DK>::kStored, stride);
      __syncthreads();
    }
  }
}

template <int DK, int DS>
__global__ void __launch_bounds__(kNT + kFetch, 1) k_delta_multiply(const Params p, const int* groups, const uint8_t* sets, int cols) {
  extern __shared__ __align__(16) uint8_t sm[];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const Job w = job_of(p, groups + 4 * blockIdx.x, blockIdx.y, blockIdx.z * cols, cols, threadIdx.x % kNT);
  const size_t stride = size_t(p.heads) * Shape<DK>::kStored;
  if (threadIdx.x < kNT) multiply<DK, 4, DS>(p, sm, w, reinterpret_cast<float*>(sm + 4 * Shape<DK>::kSet));
  else fetch_operands<DK>(p, sm, w, sets + first_set(w, blockIdx.x) * stride + size_t(w.h) * Shape<DK>::kStored, stride);
}

template <int DK>
size_t sets_bytes(const Params& p, int rows, int ngroups) { return size_t(rows / kC + ngroups + 1) * p.heads * Shape<DK>::kStored; }

template <int DK, int DS>
cudaError_t launch_multiply(const Params& p, const int* groups, const uint8_t* sets, int cols, dim3 grid, cudaStream_t st) {
  static bool done = false;
  constexpr size_t smem = 4 * Shape<DK>::kSet + (DS > 1 ? kNW * 512 * 4 : 0);
  cudaError_t e = allow_smem(k_delta_multiply<DK, DS>, smem, &done);
  return e != cudaSuccess ? e : pdl::launch(k_delta_multiply<DK, DS>, grid, dim3(kNT + kFetch), smem, st, 1, p, groups, sets, cols);
}
template <int DK>
cudaError_t launch(Params p, const int* groups, int ngroups, int rows, uint8_t* sets, bool* finished, cudaStream_t st) {
  static bool done[2] = {};
  cudaError_t e;
  if (!sets) {
    *finished = p.Vp <= kCols;
    if (*finished) p.o = nullptr;
    e = allow_smem(k_delta_chunk<DK>, Both<DK>::kBytes, &done[0]);
    return e != cudaSuccess ? e : pdl::launch(k_delta_chunk<DK>, dim3(ngroups, p.heads, (p.Vp + kCols - 1) / kCols), dim3(2 * kNT), Both<DK>::kBytes, st, 1, p, groups);
  }
  *finished = false;
  e = allow_smem(k_delta_make<DK>, Make<DK>::kBytes, &done[1]);
  const int all = rows / kC + ngroups;
  if (e == cudaSuccess) e = pdl::launch(k_delta_make<DK>, dim3((all + kMakeChunks - 1) / kMakeChunks, p.heads), dim3(kNT), Make<DK>::kBytes, st, 1, p, groups, ngroups, sets);
  if (e != cudaSuccess) return e;
  // as many CTAs per head as find room, and as many warps per 16 value columns as there are channels for: the shorter a chunk's products
  const auto ctas = [&](int cols) { return ngroups * p.heads * ((p.Vp + cols - 1) / cols); };
  int cols = kCols;
  while (cols > 16 && cols / 2 < p.Vp && ctas(cols / 2) <= tbvops::sm_count()) cols /= 2;
  const int ds = cols > 64 || DK < 64 ? 1 : (cols > 16 || DK < 128 ? 2 : 4);
  const dim3 grid(ngroups, p.heads, (p.Vp + cols - 1) / cols);
  if (ds == 1) return launch_multiply<DK, 1>(p, groups, sets, cols, grid, st);
  if constexpr (DK >= 64) {
    if (ds == 2) return launch_multiply<DK, 2>(p, groups, sets, cols, grid, st);
  }
  if constexpr (DK >= 128) return launch_multiply<DK, 4>(p, groups, sets, cols, grid, st);
  return cudaErrorInvalidValue;
}

}  // namespace

namespace delta_ops {

bool chunk_fits(const Params& p) { return p.Dp <= 128; }

size_t chunk_sets(const Params& p, int rows, int ngroups) {
  return p.Dp <= 32 ? sets_bytes<32>(p, rows, ngroups) : (p.Dp <= 64 ? sets_bytes<64>(p, rows, ngroups) : sets_bytes<128>(p, rows, ngroups));
}

cudaError_t chunk_scan(const Params& p, const int* groups, int ngroups, int rows, void* sets, bool* finished, cudaStream_t st) {
  uint8_t* s = static_cast<uint8_t*>(sets);
  if (p.Dp <= 32) return launch<32>(p, groups, ngroups, rows, s, finished, st);
  if (p.Dp <= 64) return launch<64>(p, groups, ngroups, rows, s, finished, st);
  return launch<128>(p, groups, ngroups, rows, s, finished, st);
}

}  // namespace delta_ops
