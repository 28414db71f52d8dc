// Small device helpers shared by the kernels: activation math, warp/block reductions,
// vector load/store of bf16.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace cb {

__device__ __forceinline__ float tanh_fast(float x) {
  float y;
  asm("tanh.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// tanh-approximated GELU, the constants of math::gelu in the reference
// (plugins/model-transformer/src/lib.rs:94-99).
__device__ __forceinline__ float gelu_tanh(float x) {
  const float u = 0.7978845608028654f * x * (1.0f + 0.044715f * x * x);
  return 0.5f * x * (1.0f + tanh_fast(u));
}
__device__ __forceinline__ float gelu_erf(float x) {
  return 0.5f * x * (1.0f + erff(x * 0.7071067811865476f));
}
__device__ __forceinline__ float gelu_tanh_grad(float x) {
  const float x2 = x * x;
  const float u = 0.7978845608028654f * x * (1.0f + 0.044715f * x2);
  const float t = tanh_fast(u);
  const float du = 0.7978845608028654f * (1.0f + 3.0f * 0.044715f * x2);
  return 0.5f * (1.0f + t) + 0.5f * x * (1.0f - t * t) * du;
}
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Three-input maximum and packed two-wide fp32 arithmetic (one instruction for two lanes of work;
// the softmax loops are bound by instruction issue, not by the exponential unit alone).
__device__ __forceinline__ float max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ void fma2(float& d0, float& d1, float a0, float a1, float b0, float b1,
                                     float c0, float c1) {
  asm("{\n\t.reg .b64 ra, rb, rc, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %5};\n\tmov.b64 rc, {%6, %7};\n\t"
      "fma.rn.f32x2 rd, ra, rb, rc;\n\t"
      "mov.b64 {%0, %1}, rd;\n\t}"
      : "=f"(d0), "=f"(d1) : "f"(a0), "f"(a1), "f"(b0), "f"(b1), "f"(c0), "f"(c1));
}
__device__ __forceinline__ void add2(float& d0, float& d1, float a0, float a1, float b0, float b1) {
  asm("{\n\t.reg .b64 ra, rb, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %5};\n\t"
      "add.rn.f32x2 rd, ra, rb;\n\t"
      "mov.b64 {%0, %1}, rd;\n\t}"
      : "=f"(d0), "=f"(d1) : "f"(a0), "f"(a1), "f"(b0), "f"(b1));
}
// gelu_erf of two numbers for results that are rounded to bf16, on the packed FMA units alone: on
// |x| <= L = 4.8, erf(x / sqrt 2) = x P(2 x^2 / L^2 - 1) with P of degree 11, a least-squares fit on
// Chebyshev points reweighted toward equal error.  Absolute error of the result below 4e-6 (1e-6 of
// x beyond L).
__device__ __forceinline__ void gelu_erf_pair(float& a, float& b) {
  constexpr float L = 4.8f;
  const float ca = fminf(fmaxf(a, -L), L), cb = fminf(fmaxf(b, -L), L);
  const float k = 2.0f / (L * L);
  float sa, sb, ra = -0.00129393314f, rb = -0.00129393314f;
  fma2(sa, sb, ca * k, cb * k, ca, cb, -1.0f, -1.0f);
  constexpr float P[11] = {0.294424921f, -0.145956933f, 0.105852485f, -0.0812156424f,
                           0.0609818138f, -0.0436887182f, 0.02934747f, -0.0170357972f,
                           0.00851383246f, -0.00557677634f, 0.00398022635f};
#pragma unroll
  for (int i = 10; i >= 0; --i) fma2(ra, rb, ra, rb, sa, sb, P[i], P[i]);
  const float ha = 0.5f * fmaxf(a, -L), hb = 0.5f * fmaxf(b, -L);
  fma2(a, b, ha, hb, ra * ca, rb * cb, ha, hb);
}
// Dropout masks are a pure function of (key, element index): one 32-bit hash per group of four
// consecutive elements, one byte per element; an element is dropped when its byte is below
// thr = round(p * 256), kept elements are scaled by 256 / (256 - thr).  The same function is
// restated with tensor ops on the host (ops/elementwise.py dropout_mask), so the CPU path, the
// forward pass and the recomputation in the backward pass agree bit for bit and no mask is stored.
__device__ __forceinline__ uint32_t mix32(uint32_t x) {
  x ^= x >> 16;
  x *= 0x7feb352du;
  x ^= x >> 15;
  x *= 0x846ca68bu;
  x ^= x >> 16;
  return x;
}
__device__ __forceinline__ uint32_t dropout_bits(unsigned long long group, uint32_t key) {
  return mix32(static_cast<uint32_t>(group) ^ mix32(static_cast<uint32_t>(group >> 32) ^ key));
}
// 0 for a dropped element, `scale` for a kept one: byte `lane` (0..3) of the group's hash.
__device__ __forceinline__ float dropout_factor(uint32_t bits, int lane, int thr, float scale) {
  return static_cast<int>((bits >> (8 * lane)) & 255u) < thr ? 0.f : scale;
}
__device__ __forceinline__ float silu(float x) { return x / (1.0f + __expf(-x)); }

// The gated unit of an expert: g bounded above, u on both sides, g * sigmoid(slope * g) * (u + 1).
__device__ __forceinline__ float clamped_glu(float g, float u, float slope, float limit, float shift) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return __fdividef(g * (u + shift), 1.0f + __expf(-slope * g));
}
// tanh from the fast exponential, absolute error below 3e-7
__device__ __forceinline__ float tanh_exp(float x) {
  return 1.0f - __fdividef(2.0f, 1.0f + fast_exp2(x * 2.8853900817779268f));
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Block-wide sum; `red` is a shared array of at least 32 floats.  All threads get the result.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  const int nw = (blockDim.x + 31) >> 5;
  float r = (lane < nw) ? red[lane] : 0.0f;
  r = warp_sum(r);
  return r;
}
__device__ __forceinline__ float block_max(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  const int nw = (blockDim.x + 31) >> 5;
  float r = (lane < nw) ? red[lane] : -INFINITY;
  r = warp_max(r);
  return r;
}

struct alignas(16) bf16x8 {
  __nv_bfloat162 v[4];
};
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float* f) {
  const bf16x8 x = *reinterpret_cast<const bf16x8*>(p);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 t = __bfloat1622float2(x.v[i]);
    f[2 * i] = t.x;
    f[2 * i + 1] = t.y;
  }
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float* f) {
  bf16x8 x;
#pragma unroll
  for (int i = 0; i < 4; ++i) x.v[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
  *reinterpret_cast<bf16x8*>(p) = x;
}

}  // namespace cb
