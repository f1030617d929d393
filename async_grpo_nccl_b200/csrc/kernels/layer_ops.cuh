// Shared pieces of the listed-layer kernels: Dynamic Tanh, dtype-generic loads / stores, row addressing.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace agrpo {

// tanh in 32-bit: near zero the odd Taylor series (the first dropped term is below 1e-8 of the value at |z| = 1/4), beyond
// it (1 - e) / (1 + e) with e = exp(-2 |z|), where nothing cancels any more. Used by every fused norm epilogue, so that
// all paths compute the same function whatever fast-math flags their file is built with.
__device__ __forceinline__ float tanh_f32(float z) {
  const float a = fabsf(z);
  if (a < 0.25f) {
    const float s = z * z;
    float p = 62.f / 2835.f;
    p = fmaf(p, s, -17.f / 315.f);
    p = fmaf(p, s, 2.f / 15.f);
    p = fmaf(p, s, -1.f / 3.f);
    return fmaf(z * s, p, z);
  }
  const float e = __expf(-2.f * a);
  return copysignf(__fdividef(1.f - e, 1.f + e), z);
}

// The same function for the bf16 epilogues: absolute error about 1e-7 everywhere (the difference cancels near zero), a third of
// the instructions.
__device__ __forceinline__ float tanh_abs_f32(float z) { return fmaf(-2.f, __fdividef(1.f, 1.f + __expf(2.f * z)), 1.f); }

__device__ __forceinline__ float sigmoid_f32(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

// Dynamic Tanh norm: y = tanh(alpha * x) * w + b, elementwise.
template <typename T>
struct DytNorm {
  const T* w;
  const T* b;
  const T* alpha;  // one value
};

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// eight consecutive values (16-byte aligned bf16, 32-byte run of fp32)
__device__ __forceinline__ void ld8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 w = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&w);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    v[2 * i] = f.x;
    v[2 * i + 1] = f.y;
  }
}
__device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void st8(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 w;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&w);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = w;
}
__device__ __forceinline__ void st8(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

// x[0..8) += dyt1(acc); h = dyt2(x): the tail of a sublayer (norm of its output, residual add in 32-bit, norm ahead of
// the next sublayer) on eight consecutive channels. Pointers are already offset to the row / column.
template <typename T>
__device__ __forceinline__ void dyt_residual8(const float (&acc)[8], float* x, T* h, const DytNorm<T>& n1, const DytNorm<T>& n2, int col,
                                              float a1, float a2) {
  float w1[8], b1[8], w2[8], b2[8], xv[8], hv[8];
  ld8(x, xv);
  ld8(n1.w + col, w1);
  ld8(n1.b + col, b1);
  ld8(n2.w + col, w2);
  ld8(n2.b + col, b2);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    xv[i] += fmaf(tanh_abs_f32(a1 * acc[i]), w1[i], b1[i]);
    hv[i] = fmaf(tanh_abs_f32(a2 * xv[i]), w2[i], b2[i]);
  }
  st8(x, xv);
  st8(h, hv);
}

// Where token row t of a step lives: {slot, position, first row of its segment in this step, unused}. Decode steps have
// no row table: row t is slot t at position seq_lens[t] - 1, and rows with seq_lens[t] <= 0 are idle.
struct RowMap {
  const int4* rows;
  const int* seq_lens;
  __device__ __forceinline__ int4 get(int t) const {
    if (rows != nullptr) return rows[t];
    return make_int4(t, seq_lens[t] - 1, t, 0);
  }
};

}  // namespace agrpo
