// The two tensor-core GEMMs of a parallel block: both input projections in one launch, and the output projection that adds
// mixer and feed-forward to the residual stream and prepares the next block's inputs.
#include "../common/tensormap.h"
#include "../launchers.h"
#include "gemm_tcgen05.cuh"
#include "parallel_block.cuh"

namespace agrpo {

namespace {

struct ProjEpilogue {
  ProjOut o;
  float rs, sq, sk;

  __device__ __forceinline__ void item_begin(int row, int M, int) {
    rs = o.row_scale(row, M);
    sq = sk = 0.f;
  }
  __device__ __forceinline__ void chunk(int row, int col0, const uint32_t (&r)[32], int M, int N) {
    if (row >= M) return;
#pragma unroll
    for (int c = 0; c < 32; c += 8) {
      if (col0 + c < N) {
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(r[c + i]) * rs;
        o.store8(row, col0 + c, v, sq, sk);
      }
    }
  }
  __device__ __forceinline__ void item_end(int row, int M, int, int) {
    if (row < M) o.add_stats(row, sq, sk);
  }
};

struct ResidualEpilogue {
  ResidualOut o;
  int bn;
  float sq;
  float xn[32];  // residual of the next 32 columns, read ahead

  __device__ __forceinline__ void fetch(int row, int col0, int M, int N) {
    if (row >= M || !o.accumulate) return;
    const float* src = o.x + (size_t)row * o.ldx + col0;
#pragma unroll
    for (int c = 0; c < 32; c += 4)
      if (col0 + c < N) {
        const float4 f = *reinterpret_cast<const float4*>(src + c);
        xn[c] = f.x; xn[c + 1] = f.y; xn[c + 2] = f.z; xn[c + 3] = f.w;
      }
  }
  __device__ __forceinline__ void item_begin(int, int, int) { sq = 0.f; }
  __device__ __forceinline__ void tile_begin(int row, int col0, int M, int N) { fetch(row, col0, M, N); }
  __device__ __forceinline__ void chunk(int row, int col0, const uint32_t (&r)[32], int M, int N) {
    float xv[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) xv[i] = xn[i];
    fetch(row, col0 + 32, M, col0 % bn + 32 < bn ? N : 0);
    if (row >= M) return;
#pragma unroll
    for (int c = 0; c < 32; c += 8) {
      if (col0 + c < N) {
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(r[c + i]);
        o.store8(row, col0 + c, xv + c, v, sq);
      }
    }
  }
  __device__ __forceinline__ void item_end(int row, int M, int, int) {
    if (row < M) o.add_stats(row, sq);
  }
};

struct SplitEpilogue {
  SplitOut o;

  __device__ __forceinline__ void item_begin(int, int, int) {}
  __device__ __forceinline__ void chunk(int row, int col0, const uint32_t (&r)[32], int M, int N) {
    if (row >= M) return;
#pragma unroll
    for (int c = 0; c < 32; c += 8) {
      if (col0 + c < N) {
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(r[c + i]);
        o.store8(row, col0 + c, v);
      }
    }
  }
  __device__ __forceinline__ void item_end(int, int, int, int) {}
};

template <class Epi>
void launch_tiles(const void* a, long long lda, int a_cols, const void* b, long long ldb, const GemmShape& p, const Epi& e, int BN, int num_sms,
                  cudaStream_t s) {
  const CUtensorMap ta = make_tmap_2d(a, a_cols, p.M, lda, 64, kGemmBM);
  const CUtensorMap tb = make_tmap_2d(b, p.K, p.N, ldb, 64, BN);
  if (BN == 256) gemm_launch<256, false, false>(ta, tb, p, e, num_sms, s);
  else if (BN == 128) gemm_launch<128, false, false>(ta, tb, p, e, num_sms, s);
  else if (BN == 64) gemm_launch<64, false, false>(ta, tb, p, e, num_sms, s);
  else gemm_launch<32, false, false>(ta, tb, p, e, num_sms, s);
}

int pick_bn(const GemmShape& p) {  // widest column tile that still gives about one work item per SM
  const int cands[3] = {256, 128, 64};
  for (int bn : cands)
    if (gemm_num_items(p.M, p.N, bn, 1, p.n1) >= 120) return bn;
  return 32;
}

}  // namespace

void launch_gemm_parallel_proj(const ParallelProjArgs& a, int num_sms, cudaStream_t s) {
  if (a.M == 0) return;
  const ProjOut out = proj_out(a);
  if (launch_gemm_skinny_proj(a, out, num_sms, s)) return;
  GemmShape p;
  p.M = a.M; p.N = a.n1 + a.n2; p.K = a.K;
  p.group_n = 1;
  p.status = a.status;
  p.n1 = a.n2 > 0 ? a.n1 : 0;
  p.a2 = a.a2;
  ProjEpilogue e;
  e.o = out;
  e.rs = 1.f;
  e.sq = e.sk = 0.f;
  launch_tiles(a.h, a.lda, a.n2 > 0 ? a.a2 + a.K : a.K, a.w, a.ldw, p, e, pick_bn(p), num_sms, s);
}

void launch_gemm_residual(const ResidualArgs& a, int num_sms, cudaStream_t s) {
  if (a.M == 0) return;
  const ResidualOut out = residual_out(a);
  if (launch_gemm_skinny_residual(a, out, num_sms, s)) return;
  GemmShape p;
  p.M = a.M; p.N = a.N; p.K = a.K;
  p.group_n = 1;
  p.status = a.status;
  ResidualEpilogue e;
  e.o = out;
  e.sq = 0.f;
  e.bn = pick_bn(p);
  launch_tiles(a.a, a.lda, a.K, a.w, a.ldw, p, e, e.bn, num_sms, s);
}

void launch_gemm_split_store(const SplitStoreArgs& a, int num_sms, cudaStream_t s) {
  if (a.M == 0) return;
  const SplitOut out = split_out(a);
  if (launch_gemm_skinny_split(a, out, num_sms, s)) return;
  GemmShape p;
  p.M = a.M; p.N = a.n1 + a.n2; p.K = a.K;
  p.group_n = 1;
  p.status = a.status;
  launch_tiles(a.a, a.lda, a.K, a.w, a.ldw, p, SplitEpilogue{out}, pick_bn(p), num_sms, s);
}

}  // namespace agrpo
