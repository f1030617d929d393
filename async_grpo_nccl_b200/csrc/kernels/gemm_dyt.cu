// Tensor-core GEMM whose epilogue is the tail of a sublayer: the output's Dynamic Tanh norm, the fp32 residual add and the
// norm ahead of the next sublayer. The norms are elementwise, so nothing between two GEMMs needs a pass of its own.
#include "../common/tensormap.h"
#include "../launchers.h"
#include "../launchers_layers.h"
#include "gemm_tcgen05.cuh"
#include "layer_ops.cuh"

namespace agrpo {

namespace {

struct DytResidualEpilogue {
  float* x;              // [M, ldx] fp32 residual stream, updated in place
  long long ldx;
  __nv_bfloat16* h;      // [M, ldh] input of the next sublayer
  long long ldh;
  DytNorm<__nv_bfloat16> n1, n2;
  float a1, a2;
  int bn;                // column tile of the kernel
  float xn[32];          // residual of the next 32 columns, read ahead

  // 32 residual values of one row; columns past N (a multiple of 8) are not read
  __device__ __forceinline__ void fetch(int row, int col0, int M, int N) {
    if (row >= M) return;
    const float* src = x + (size_t)row * ldx + col0;
#pragma unroll
    for (int c = 0; c < 32; c += 4)
      if (col0 + c < N) {
        const float4 f = *reinterpret_cast<const float4*>(src + c);
        xn[c] = f.x; xn[c + 1] = f.y; xn[c + 2] = f.z; xn[c + 3] = f.w;
      }
  }
  __device__ __forceinline__ void item_begin(int, int, int) {
    a1 = ldf(n1.alpha);
    a2 = ldf(n2.alpha);
  }
  __device__ __forceinline__ void tile_begin(int row, int col0, int M, int N) { fetch(row, col0, M, N); }
  __device__ __forceinline__ void item_end(int, int, int, int) {}
  __device__ __forceinline__ void chunk(int row, int col0, const uint32_t (&r)[32], int M, int N) {
    float xv[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) xv[i] = xn[i];
    fetch(row, col0 + 32, M, col0 % bn + 32 < bn ? N : 0);  // within the tile: the next tile's rows are read by tile_begin
    if (row >= M || col0 >= N) return;
    float* xd = x + (size_t)row * ldx + col0;
    __nv_bfloat16* hd = h + (size_t)row * ldh + col0;
#pragma unroll
    for (int c = 0; c < 32; c += 8) {
      if (col0 + c < N) {
        float w1[8], b1[8], w2[8], b2[8], xo[8], ho[8];
        ld8(n1.w + col0 + c, w1);
        ld8(n1.b + col0 + c, b1);
        ld8(n2.w + col0 + c, w2);
        ld8(n2.b + col0 + c, b2);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          xo[i] = xv[c + i] + fmaf(tanh_abs_f32(a1 * __uint_as_float(r[c + i])), w1[i], b1[i]);
          ho[i] = fmaf(tanh_abs_f32(a2 * xo[i]), w2[i], b2[i]);
        }
        st8(xd + c, xo);
        st8(hd + c, ho);
      }
    }
  }
};

}  // namespace

void launch_gemm_dyt_bf16(const void* a, long long lda, const void* b, long long ldb, int M, int N, int K, float* x, long long ldx, void* h,
                          long long ldh, const DytArgs& n1, const DytArgs& n2, int* status, int num_sms, cudaStream_t s) {
  if (M == 0 || N == 0) return;
  const DytTail tail{x, ldx, h, ldh, n1, n2};
  if (M <= 256 && launch_gemm_skinny(a, lda, b, ldb, nullptr, 0, M, N, K, nullptr, nullptr, 0, status, num_sms, s, nullptr, nullptr, nullptr, 0.f,
                                     nullptr, &tail))
    return;
  const int tiles_m = (M + kGemmBM - 1) / kGemmBM;
  const int cands[3] = {256, 128, 64};
  int BN = 32;
  for (int bn : cands)
    if ((long long)tiles_m * ((N + bn - 1) / bn) >= 120) {
      BN = bn;
      break;
    }
  const CUtensorMap ta = make_tmap_2d(a, K, M, lda, 64, kGemmBM);
  const CUtensorMap tb = make_tmap_2d(b, K, N, ldb, 64, BN);
  GemmShape p;
  p.M = M; p.N = N; p.K = K;
  p.group_n = 1;
  p.status = status;
  DytResidualEpilogue e;
  e.x = x;
  e.ldx = ldx;
  e.h = reinterpret_cast<__nv_bfloat16*>(h);
  e.ldh = ldh;
  typedef const __nv_bfloat16* P;
  e.n1 = {(P)n1.w, (P)n1.b, (P)n1.alpha};
  e.n2 = {(P)n2.w, (P)n2.b, (P)n2.alpha};
  e.a1 = e.a2 = 0.f;
  e.bn = BN;
  if (BN == 256) gemm_launch<256, false, false>(ta, tb, p, e, num_sms, s);
  else if (BN == 128) gemm_launch<128, false, false>(ta, tb, p, e, num_sms, s);
  else if (BN == 64) gemm_launch<64, false, false>(ta, tb, p, e, num_sms, s);
  else gemm_launch<32, false, false>(ta, tb, p, e, num_sms, s);
}

}  // namespace agrpo
