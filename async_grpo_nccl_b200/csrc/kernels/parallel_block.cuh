// Epilogues of the two GEMMs of a parallel block (mixer and feed-forward read the same residual stream and are added to it
// together), shared by the persistent and the split-K kernels.
//
// No norm runs as a kernel of its own. A zero-centred RMS norm is x * (1 + w) times a row scale: the GEMM that produces x writes
// x * (1 + w) (bf16 rounding does not depend on the scale) and adds up the squares of its rows, the GEMM that consumes it
// multiplies its rows by 1 / sqrt(mean + eps).
#pragma once
#include "../common/ptx.cuh"
#include "../launchers_hybrid.h"
#include "layer_ops.cuh"

namespace agrpo {

// u = first product, act = relu(second product)^2; see ParallelProjArgs.
struct ProjOut {
  __nv_bfloat16* u;     // nullptr = off
  long long ldu;
  __nv_bfloat16* act;
  long long ldact;
  int n1;
  const sumsq_t* ss_in;
  float inv_w, eps;
  sumsq_t* ss_q;
  sumsq_t* ss_k;
  int q_end, k_end;

  __device__ __forceinline__ float row_scale(int row, int M) const {
    return ss_in != nullptr && row < M ? rsqrtf(sumsq_from_fixed(ss_in[row]) * inv_w + eps) : 1.f;
  }
  // eight columns of one row, already scaled; n1 and the number of columns are multiples of 8
  __device__ __forceinline__ void store8(int row, int col, float (&v)[8], float& sq, float& sk) const {
    if (col < n1) {
      if (col < k_end) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) s += v[i] * v[i];
        if (col < q_end) sq += s;
        else sk += s;
      }
      st8(u + (size_t)row * ldu + col, v);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float z = fmaxf(v[i], 0.f);
        v[i] = z * z;
      }
      st8(act + (size_t)row * ldact + (col - n1), v);
    }
  }
  __device__ __forceinline__ void add_stats(int row, float sq, float sk) const {
    if (ss_q == nullptr) return;
    if (sq != 0.f) sumsq_atomic_add(ss_q + row, sq);
    if (sk != 0.f) sumsq_atomic_add(ss_k + row, sk);
  }
};

inline ProjOut proj_out(const ParallelProjArgs& a) {
  ProjOut o;
  o.u = reinterpret_cast<__nv_bfloat16*>(a.u);
  o.ldu = a.ldu;
  o.act = reinterpret_cast<__nv_bfloat16*>(a.act);
  o.ldact = a.ldact;
  o.n1 = a.n1;
  o.ss_in = a.ss_in;
  o.inv_w = 1.f / (float)a.width;
  o.eps = a.eps;
  o.ss_q = a.ss_q;
  o.ss_k = a.ss_k;
  o.q_end = a.ss_q != nullptr ? a.q_end : 0;
  o.k_end = a.ss_q != nullptr ? a.k_end : 0;
  return o;
}

// x (+)= product on the fp32 stream, its consumers and its sums of squares; see ResidualArgs.
struct ResidualOut {
  float* x;             // nullptr = off
  long long ldx;
  int accumulate;
  __nv_bfloat16* h[2];
  long long ldh[2];
  const __nv_bfloat16* w[2];
  sumsq_t* ss;

  // eight columns of one row; x0 = the old values (ignored unless accumulating)
  __device__ __forceinline__ void store8(int row, int col, const float* x0, float (&v)[8], float& sq) const {
    if (accumulate) {
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] += x0[i];
    }
    if (ss != nullptr) {
#pragma unroll
      for (int i = 0; i < 8; ++i) sq += v[i] * v[i];
    }
    st8(x + (size_t)row * ldx + col, v);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      if (h[k] == nullptr) continue;
      float y[8];
      if (w[k] != nullptr) {
        ld8(w[k] + col, y);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = fmaf(v[i], y[i], v[i]);
        st8(h[k] + (size_t)row * ldh[k] + col, y);
      } else {
        st8(h[k] + (size_t)row * ldh[k] + col, v);
      }
    }
  }
  __device__ __forceinline__ void add_stats(int row, float sq) const {
    if (ss != nullptr) sumsq_atomic_add(ss + row, sq);
  }
};

inline ResidualOut residual_out(const ResidualArgs& a) {
  ResidualOut o;
  o.x = a.x;
  o.ldx = a.ldx;
  o.accumulate = a.accumulate;
  for (int k = 0; k < 2; ++k) {
    o.h[k] = reinterpret_cast<__nv_bfloat16*>(a.out[k].h);
    o.ldh[k] = a.out[k].ld;
    o.w[k] = reinterpret_cast<const __nv_bfloat16*>(a.out[k].w);
  }
  o.ss = a.ss;
  return o;
}

// First n1 columns as bf16, the others as fp32; see SplitStoreArgs.
struct SplitOut {
  __nv_bfloat16* d16;   // nullptr = off
  long long ld16;
  float* d32;
  long long ld32;
  int n1;
  __device__ __forceinline__ void store8(int row, int col, const float (&v)[8]) const {
    if (col < n1) st8(d16 + (size_t)row * ld16 + col, v);
    else st8(d32 + (size_t)row * ld32 + (col - n1), v);
  }
};
inline SplitOut split_out(const SplitStoreArgs& a) {
  return SplitOut{reinterpret_cast<__nv_bfloat16*>(a.d16), a.ld16, a.d32, a.ld32, a.n1};
}

// Split-K forms (gemm_splitk.cu) for up to 256 rows; false when the shape is not served.
bool launch_gemm_skinny_proj(const ParallelProjArgs& a, const ProjOut& out, int num_sms, cudaStream_t s);
bool launch_gemm_skinny_split(const SplitStoreArgs& a, const SplitOut& out, int num_sms, cudaStream_t s);
bool launch_gemm_skinny_residual(const ResidualArgs& a, const ResidualOut& out, int num_sms, cudaStream_t s);

}  // namespace agrpo
