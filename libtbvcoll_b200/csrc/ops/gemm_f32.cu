// gemm_f32.cu — full 32-bit GEMM on the CUDA cores, for models run with fp32 weights and activations (numerics
// checks; tensor cores have no full-fp32 mode).  Same epilogues and grouped form as the tcgen05 GEMM's extended entry.
//
//   y[n, m] = epilogue(sum_k x[n, k] * w[m, k])        x: [N, K], w: [groups * M, K], fp32 row-major
//
// 64 tokens x 64 features per CTA, K in steps of 16 through shared memory, 4 x 4 outputs per thread.  The order of
// the additions for one output depends on K alone, so a row's result does not depend on the batch it is in.
#include <cuda_runtime.h>

#include "gemm.cuh"

namespace {

constexpr int kT = 64, kKB = 16;

struct F32Params {
  const float *w, *x, *bias;
  float* y;
  int M, N, K, ldx, ldy, epi, act, groups, x_group, y_group;
  float act_a, act_b, act_c;
  int m_last;             // > 0: one more group with this many features
  int act_m;              // the activation acts on the first act_m features
  const int* row_off;     // row-grouped form: group g owns rows row_off[g] .. row_off[g + 1] - 1
};

__global__ void __launch_bounds__(256) k_gemm_f32(const F32Params p) {
  __shared__ float sx[kKB][kT + 4], sw[kKB][kT + 4];
  pdl::launch_dependents();
  pdl::grid_dependency_wait();
  const int mt = (p.M + kT - 1) / kT, grp = min(int(blockIdx.x) / mt, p.m_last ? p.groups : p.groups - 1);
  const int m0 = (blockIdx.x - grp * mt) * kT, M = p.m_last && grp == p.groups ? p.m_last : p.M;
  int n0 = blockIdx.y * kT, nend = p.N;
  if (p.row_off) {
    nend = p.row_off[grp + 1];
    n0 += p.row_off[grp];
    if (n0 >= nend) return;
  }
  const float* w = p.w + size_t(grp) * p.M * p.K;
  const float* x = p.x + size_t(grp) * p.x_group;
  float* y = p.y + size_t(grp) * p.y_group;
  const int tm = (threadIdx.x & 15) * 4, tn = (threadIdx.x >> 4) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += kKB) {
    for (int i = threadIdx.x; i < kT * kKB; i += 256) {
      const int r = i / kKB, k = i % kKB;
      sx[k][r] = (n0 + r < nend && k0 + k < p.K) ? x[size_t(n0 + r) * p.ldx + k0 + k] : 0.f;
      sw[k][r] = (m0 + r < M && k0 + k < p.K) ? w[size_t(m0 + r) * p.K + k0 + k] : 0.f;
    }
    __syncthreads();
    float part[4][4] = {};      // one step's sum apart from the running total: the rounding error grows with K / 16, not with K
#pragma unroll
    for (int k = 0; k < kKB; k++) {
      const float4 a = *reinterpret_cast<const float4*>(&sx[k][tn]), b = *reinterpret_cast<const float4*>(&sw[k][tm]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) part[i][j] = fmaf(av[i], bv[j], part[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
      for (int j = 0; j < 4; j++) acc[i][j] += part[i][j];
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int n = n0 + tn + i;
    if (n >= nend) continue;
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; j++) v[j] = acc[i][j] + ((p.bias && m0 + tm + j < M) ? p.bias[m0 + tm + j] : 0.f);
    if (p.epi == gemm::kEpiClampGlu) {
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        if (m0 + tm + j + 1 < M) {
          const float g = fminf(v[j], p.act_a), u = fminf(fmaxf(v[j + 1], -p.act_a), p.act_a);
          y[size_t(n) * p.ldy + (m0 + tm + j) / 2] = (isinf(p.act_b) ? fmaxf(g, 0.f) : g / (1.0f + expf(-p.act_b * g))) * (u + p.act_c);
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < 4; j++)
        if (m0 + tm + j < M) {
          if (p.act && m0 + tm + j < p.act_m) {
            if (p.act == gemm::kActSilu || p.act == gemm::kActGelu) v[j] = v[j] / (1.0f + expf(p.act == gemm::kActSilu ? -v[j] : -gemm::gelu_slope(v[j])));
            else v[j] = p.act == gemm::kActSoftplus ? vec::softplus<float>(v[j]) : gemm::apply_act(v[j], p.act, p.act_a);
          }
          y[size_t(n) * p.ldy + m0 + tm + j] = v[j];
        }
    }
  }
}

}  // namespace

extern "C" {

// Arguments as tbv_op_gemm_ex, everything fp32; epi 0 / 2 store (act applies), 3 clamped gated unit.
int tbv_op_gemm_f32(const void* w, const void* x, void* y, const void* bias, int M, int N, int K, int ldx, int ldy, int epi, int act,
                    float act_a, float act_b, float act_c, int act_m, int groups, int x_group, int y_group, int m_last, void* stream) {
  if (M <= 0 || N <= 0 || K <= 0 || (epi != 0 && epi != 2 && epi != 3) || (epi == 3 && (M % 2)) || (groups > 1 && bias)) return -2;
  F32Params p{static_cast<const float*>(w), static_cast<const float*>(x), static_cast<const float*>(bias), static_cast<float*>(y),
              M, N, K, ldx, ldy, epi, act, groups > 1 ? groups : 1, x_group, y_group, act_a, act_b, act_c, groups > 1 ? m_last : 0, act_m, nullptr};
  const dim3 grid(p.groups * ((M + kT - 1) / kT) + (p.m_last + kT - 1) / kT, (N + kT - 1) / kT);
  return pdl::launch(k_gemm_f32, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), 1, p) == cudaSuccess ? 0 : -1;
}

// Arguments as tbv_op_gemm_rows, everything fp32.
int tbv_op_gemm_rows_f32(const void* w, const void* x, void* y, const void* row_off, int groups, int M, int x_rows, int max_rows, int K, int ldx,
                         int ldy, int epi, float act_a, float act_b, float act_c, void* stream) {
  if (M <= 0 || x_rows <= 0 || max_rows <= 0 || K <= 0 || groups <= 0 || (epi != 0 && epi != 3) || (epi == 3 && (M % 2)) || !row_off) return -2;
  F32Params p{static_cast<const float*>(w), static_cast<const float*>(x), nullptr, static_cast<float*>(y),
              M, max_rows, K, ldx, ldy, epi, 0, groups, 0, 0, act_a, act_b, act_c, 0, 0, static_cast<const int*>(row_off)};
  const dim3 grid(groups * ((M + kT - 1) / kT), (max_rows + kT - 1) / kT);
  return pdl::launch(k_gemm_f32, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), 1, p) == cudaSuccess ? 0 : -1;
}

}  // extern "C"
