// vec.cuh — small helpers of the kernels that run on bf16 or fp32 activations: conversions, eight-wide loads and stores, SiLU, sigmoid, softplus,
// angles, and packed pairs of fp32 values.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace vec {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void from_f(float& d, float v) { d = v; }
__device__ __forceinline__ void from_f(__nv_bfloat16& d, float v) { d = __float2bfloat16_rn(v); }
__device__ __forceinline__ float silu(float v) { return v / (1.0f + expf(-v)); }
// SiLU: bf16 models take the fast exponential and division (1 + e^-v may overflow to infinity: the quotient is 0)
template <typename T> __device__ __forceinline__ float gate(float v);
template <> __device__ __forceinline__ float gate<float>(float v) { return silu(v); }
template <> __device__ __forceinline__ float gate<__nv_bfloat16>(float v) { return __fdividef(v, 1.0f + __expf(-v)); }

template <typename T> __device__ __forceinline__ float sigmoid(float v);
template <> __device__ __forceinline__ float sigmoid<float>(float v) { return 1.0f / (1.0f + expf(-v)); }
template <> __device__ __forceinline__ float sigmoid<__nv_bfloat16>(float v) { return __fdividef(1.0f, 1.0f + __expf(-v)); }

// log(1 + e^v), relative error near 2^-21 also where it is tiny.  fp32 models: CUDA's functions.  bf16 models: max(v, 0) + log1p(e^-|v|)
// with log1p(e) = 2 atanh(e / (2 + e)), whose series in the square of e / (2 + e) <= 1/3 is cut after the 15th power.
template <typename T> __device__ __forceinline__ float softplus(float v);
template <> __device__ __forceinline__ float softplus<float>(float v) { return v > 20.f ? v : log1pf(expf(v)); }
template <> __device__ __forceinline__ float softplus<__nv_bfloat16>(float v) {
  const float e = __expf(-fabsf(v)), r = __fdividef(e, 2.f + e), q = r * r;
  float h = 1.f / 15.f;
  h = fmaf(h, q, 1.f / 13.f);
  h = fmaf(h, q, 1.f / 11.f);
  h = fmaf(h, q, 1.f / 9.f);
  h = fmaf(h, q, 1.f / 7.f);
  h = fmaf(h, q, 1.f / 5.f);
  h = fmaf(h, q, 1.f / 3.f);
  h = fmaf(h, q, 1.f);
  return fmaxf(v, 0.f) + 2.f * r * h;
}
// 2^x: the hardware instruction for bf16 models, CUDA's exp2f for fp32 ones
template <typename T> __device__ __forceinline__ float pow2(float x);
template <> __device__ __forceinline__ float pow2<float>(float x) { return exp2f(x); }
template <> __device__ __forceinline__ float pow2<__nv_bfloat16>(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ void load8(const float* p, float* f) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float* f) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
  f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
  f[4] = __uint_as_float(v.z << 16); f[5] = __uint_as_float(v.z & 0xffff0000u);
  f[6] = __uint_as_float(v.w << 16); f[7] = __uint_as_float(v.w & 0xffff0000u);
}
// eight channels as they lie in memory
template <typename T> struct Raw8;
template <> struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = a; *reinterpret_cast<float4*>(p + 4) = b; }
  __device__ __forceinline__ void load(const float* p) { a = *reinterpret_cast<const float4*>(p); b = *reinterpret_cast<const float4*>(p + 4); }
  __device__ __forceinline__ void unpack(float* f) const { f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w; }
};
template <> struct Raw8<__nv_bfloat16> {
  uint4 v;
  __device__ __forceinline__ void store(__nv_bfloat16* p) const { *reinterpret_cast<uint4*>(p) = v; }
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void unpack(float* f) const {
    f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
    f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
    f[4] = __uint_as_float(v.z << 16); f[5] = __uint_as_float(v.z & 0xffff0000u);
    f[6] = __uint_as_float(v.w << 16); f[7] = __uint_as_float(v.w & 0xffff0000u);
  }
};
__device__ __forceinline__ void store8(float* p, const float* f) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float* f) {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; i++) {
    __nv_bfloat162 v = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
    w[i] = *reinterpret_cast<uint32_t*>(&v);
  }
  *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}

// sine and cosine of position * 2 pi * f, f = hi + lo turns per position; the angle is reduced before it is rounded
__device__ __forceinline__ void sincos_turns(float pos, float2 f, float* s, float* c) {
  const float t = pos * f.x, e = fmaf(pos, f.x, -t);      // t + e is the exact product
  const float frac = (t - rintf(t)) + fmaf(pos, f.y, e);
  sincospif(2.0f * frac, s, c);
}

// Two fp32 values in a 64-bit register pair: one instruction does both (each rounded as its scalar form).
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}

}  // namespace vec
