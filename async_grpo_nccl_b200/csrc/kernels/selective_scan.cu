// Selective scan (Mamba) in one kernel after the narrow projection of its input: step sizes on the tensor cores, softplus,
// decays, recurrence, read-out, skip and gate. The state lives in registers while a segment runs and in fp32 memory in between.
//
// Every (token, channel, state) needs one exponential, and the recurrence itself is sequential in time, so the kernel is laid
// out for the exponential units: four lanes share a channel, NS states each, 32 channels per CTA, and a segment's tokens go
// through shared memory in tiles that are loaded one ahead. Step sizes of a tile are a small matrix product with the channel
// block's rows of W_dt, done by mma.sync in place, so that they never exist in memory (they would be as large as the input in
// fp32). Read-outs of four tokens are summed over the four lanes at once: three shuffles, after which each lane finishes one.
//
// The projection of the input arrives as the step-size code, bf16 rows of rank_p values (a multiple of 16) eight more apart, and B
// and C, fp32 [T, 8 NS]: for each quarter of the states NS values of B, then NS of C. Both are copied to shared memory as they are. A in log2 units [C, 4 NS]; state [slots, C, 4 NS].
#include <cuda_bf16.h>

#include "../common/ptx.cuh"
#include "../launchers.h"
#include "../launchers_hybrid.h"
#include "decode_attn.cuh"
#include "layer_ops.cuh"

namespace agrpo {

namespace {

typedef __nv_bfloat16 bf16;
typedef unsigned long long f32x2;

constexpr int kCh = 32;        // channels per CTA
constexpr int kScanThreads = 128;
constexpr int kYPitch = kCh + 4;   // floats per token of the read-outs

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// ln(1 + e^v) = max(v, 0) + ln(1 + e) with e = exp(-|v|) <= 1, and ln(1 + e) = 2 artanh(e / (2 + e)): the argument is at most 1/3,
// where the odd series converges by 1/9 a term (the first one left out is below 1e-9 of the sum). Two at a time.
__device__ __forceinline__ void softplus_pair(float v0, float v1, float& r0, float& r1) {
  const float e0 = __expf(-fabsf(v0)), e1 = __expf(-fabsf(v1));
  const f32x2 s = pack2(__fdividef(e0, 2.f + e0), __fdividef(e1, 2.f + e1));
  const f32x2 q = mul2(s, s);
  f32x2 p = pack2(1.f / 17.f, 1.f / 17.f);
  p = fma2(p, q, pack2(1.f / 15.f, 1.f / 15.f));
  p = fma2(p, q, pack2(1.f / 13.f, 1.f / 13.f));
  p = fma2(p, q, pack2(1.f / 11.f, 1.f / 11.f));
  p = fma2(p, q, pack2(1.f / 9.f, 1.f / 9.f));
  p = fma2(p, q, pack2(1.f / 7.f, 1.f / 7.f));
  p = fma2(p, q, pack2(1.f / 5.f, 1.f / 5.f));
  p = fma2(p, q, pack2(1.f / 3.f, 1.f / 3.f));
  p = fma2(p, q, pack2(1.f, 1.f));
  p = fma2(mul2(s, pack2(2.f, 2.f)), p, pack2(fmaxf(v0, 0.f), fmaxf(v1, 0.f)));
  unpack2(p, r0, r1);
}

struct ScanSizes {
  int rank_p, cpitch;     // step-size code: columns, bf16 elements per row in shared memory (also of W_dt's rows)
  int bc;                 // B and C: floats per row
};
inline ScanSizes scan_sizes(int rank, int ns) {
  ScanSizes z;
  z.rank_p = (rank + 15) / 16 * 16;
  z.cpitch = scan_code_pitch(rank);
  z.bc = 8 * ns;
  return z;
}
// A stage holds tt tokens: code, B and C, x, z (kCh channels each)
__host__ __device__ inline int scan_stage_bytes(const ScanSizes& z, int tt) { return tt * (z.cpitch * 2 + z.bc * 4 + 2 * kCh * 2); }
inline int scan_smem_bytes(const ScanSizes& z, int tt, int stages) {
  return stages * scan_stage_bytes(z, tt) + kCh * z.cpitch * 2 + tt * (kCh * 16 + kYPitch * 4);
}
template <int TT>
struct Stage {
  bf16* code;
  float* bc;
  bf16* x;
  bf16* z;
  __device__ __forceinline__ Stage(uint8_t* base, const ScanSizes& s)
      : code(reinterpret_cast<bf16*>(base)), bc(reinterpret_cast<float*>(base + TT * s.cpitch * 2)),
        x(reinterpret_cast<bf16*>(base + TT * (s.cpitch * 2 + s.bc * 4))), z(x + TT * kCh) {}
};

__device__ __forceinline__ void load_wdt(const ScanArgs& p, const ScanSizes& z, int c0, bf16* sw) {  // completes with the first tile
  for (int c = threadIdx.x >> 5; c < kCh; c += 4)
    for (int k = (threadIdx.x & 31) * 8; k < z.rank_p; k += 256) {
      if (c0 + c < p.C) cp_async16(sw + c * z.cpitch + k, reinterpret_cast<const bf16*>(p.wdt) + (size_t)(c0 + c) * p.ldw + k);
      else *reinterpret_cast<uint4*>(sw + c * z.cpitch + k) = make_uint4(0u, 0u, 0u, 0u);
    }
}

// Tile rows [0, n) into a stage. Rows of the code, B and C from n on become zeros: their tokens are computed like the others, with a
// step size of zero, and must find finite numbers.
template <int TT>
__device__ __forceinline__ void load_tile(const ScanArgs& p, const ScanSizes& z, int row0, int n, int c0, const Stage<TT>& st) {
  const uint8_t* code = reinterpret_cast<const uint8_t*>(p.code) + (size_t)row0 * z.cpitch * 2;
  const uint8_t* bc = reinterpret_cast<const uint8_t*>(p.r + (size_t)row0 * z.bc);
  const int n_code = n * z.cpitch / 8, n_bc = n * z.bc / 4;   // rows lie one after the other: flat copies of 16-byte pieces
  for (int i = threadIdx.x; i < n_code; i += kScanThreads) cp_async16(reinterpret_cast<uint8_t*>(st.code) + i * 16, code + (size_t)i * 16);
  for (int i = threadIdx.x; i < n_bc; i += kScanThreads) cp_async16(reinterpret_cast<uint8_t*>(st.bc) + i * 16, bc + (size_t)i * 16);
  if (n < TT) {
    for (int i = n_code + threadIdx.x; i < TT * z.cpitch / 8; i += kScanThreads) reinterpret_cast<uint4*>(st.code)[i] = make_uint4(0u, 0u, 0u, 0u);
    for (int i = n_bc + threadIdx.x; i < TT * z.bc / 4; i += kScanThreads) reinterpret_cast<uint4*>(st.bc)[i] = make_uint4(0u, 0u, 0u, 0u);
  }
  for (int i = threadIdx.x; i < n * 4; i += kScanThreads) {
    const int t = i >> 2, k = (i & 3) * 8;
    if (c0 + k < p.C) {
      cp_async16(st.x + t * kCh + k, reinterpret_cast<const bf16*>(p.xc) + (size_t)(row0 + t) * p.ldx + c0 + k);
      cp_async16(st.z + t * kCh + k, reinterpret_cast<const bf16*>(p.z) + (size_t)(row0 + t) * p.ldz + c0 + k);
    }
  }
}

// {dt, dt, dt x, dt x} of TT tokens x 32 channels (each twice, as operands of paired arithmetic); tokens from n on get zeros, which leave a state as it is. Warp = 8 channels.
template <int TT>
__device__ __forceinline__ void step_sizes(const ScanSizes& z, const Stage<TT>& st, const bf16* sw, const float (&bias)[2], int n, float4* sdt) {
  constexpr int M = TT / 16;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, q2 = (lane & 3) * 2;
  float acc[M][4];
#pragma unroll
  for (int m = 0; m < M; ++m)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[m][e] = 0.f;
  const bf16* arow = st.code + (lane & 15) * z.cpitch + (lane >> 4) * 8;
  const bf16* wrow = sw + (warp * 8 + g) * z.cpitch + q2;
  for (int k = 0; k < z.rank_p; k += 16) {
    const uint32_t b0 = *reinterpret_cast<const uint32_t*>(wrow + k), b1 = *reinterpret_cast<const uint32_t*>(wrow + k + 8);
#pragma unroll
    for (int m = 0; m < M; ++m) {
      uint32_t a[4];
      ldmatrix_x4(a, arow + m * 16 * z.cpitch + k);
      mma_16816(acc[m], a[0], a[1], a[2], a[3], b0, b1);
    }
  }
#pragma unroll
  for (int m = 0; m < M; ++m)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int t = m * 16 + g + (e >> 1) * 8, c = warp * 8 + q2;
      float d0 = 0.f, d1 = 0.f;
      float2 x = make_float2(0.f, 0.f);
      if (t < n) {
        x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(st.x + t * kCh + c));
        softplus_pair(acc[m][e] + bias[0], acc[m][e + 1] + bias[1], d0, d1);
      }
      sdt[t * kCh + c] = make_float4(d0, d0, d0 * x.x, d0 * x.x);
      sdt[t * kCh + c + 1] = make_float4(d1, d1, d1 * x.y, d1 * x.y);
    }
}

// Decays exp2(dt A) of one token of one channel quarter.
template <int NS>
__device__ __forceinline__ void scan_decays(const f32x2 dt, const f32x2 (&A)[NS / 2], f32x2 (&e)[NS / 2]) {
#pragma unroll
  for (int i = 0; i < NS / 2; ++i) {
    float a, b;
    unpack2(mul2(dt, A[i]), a, b);
    e[i] = pack2(ex2(a), ex2(b));
  }
}

// The token itself: S <- e S + (dt x) B; returns this quarter's part of S . C.
template <int NS>
__device__ __forceinline__ float scan_update(const f32x2 dx, const float* bc, const f32x2 (&e)[NS / 2], f32x2 (&S)[NS / 2]) {
  f32x2 B[NS / 2], C[NS / 2];
  if constexpr (NS >= 4) {
#pragma unroll
    for (int i = 0; i < NS / 4; ++i) {
      const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(bc + 4 * i), c = *reinterpret_cast<const ulonglong2*>(bc + NS + 4 * i);
      B[2 * i] = b.x; B[2 * i + 1] = b.y;
      C[2 * i] = c.x; C[2 * i + 1] = c.y;
    }
  } else {
    const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(bc);
    B[0] = v.x;
    C[0] = v.y;
  }
  f32x2 y = 0;
#pragma unroll
  for (int i = 0; i < NS / 2; ++i) {
    S[i] = fma2(e[i], S[i], mul2(dx, B[i]));
    y = i == 0 ? mul2(S[i], C[i]) : fma2(S[i], C[i], y);
  }
  float a, b;
  unpack2(y, a, b);
  return a + b;
}

template <int NS>
__device__ __forceinline__ float scan_step(const float4* d, const float* bc, const f32x2 (&A)[NS / 2], f32x2 (&S)[NS / 2]) {
  const ulonglong2 dd = *reinterpret_cast<const ulonglong2*>(d);
  f32x2 e[NS / 2];
  scan_decays<NS>(dd.x, A, e);
  return scan_update<NS>(dd.y, bc, e, S);
}

// Sums over the four lanes of a channel for four tokens: lane q gets token q.
__device__ __forceinline__ float quad_transpose_sum(const float (&y)[4], int q) {
  const bool odd = q & 1, high = q & 2;
  float a = odd ? y[1] : y[0], b = odd ? y[3] : y[2];
  a += __shfl_xor_sync(0xffffffffu, odd ? y[0] : y[1], 1);
  b += __shfl_xor_sync(0xffffffffu, odd ? y[2] : y[3], 1);
  return (high ? b : a) + __shfl_xor_sync(0xffffffffu, high ? a : b, 2);
}

// Finished read-outs of a tile -> skip, gate, store: thread = 8 channels of a token.
template <int TT>
__device__ __forceinline__ void store_tile(const ScanArgs& p, const Stage<TT>& st, const float* sy, const float* sskip, size_t row0, int n, int c0,
                                           const int* s_pos) {
  for (int i = threadIdx.x; i < n * 4; i += kScanThreads) {
    const int t = i >> 2, k = (i & 3) * 8;
    if (c0 + k >= p.C || (s_pos != nullptr && s_pos[t] < 0)) continue;
    float x[8], z[8], d[8], o[8];
    ld8(st.x + t * kCh + k, x);
    ld8(st.z + t * kCh + k, z);
    ld8(sskip + k, d);
    ld8(sy + t * kYPitch + k, o);
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] = fmaf(d[e], x[e], o[e]) * z[e] * sigmoid_f32(z[e]);
    st8(reinterpret_cast<bf16*>(p.out) + (row0 + t) * p.ldo + c0 + k, o);
  }
}

// Per-thread constants of a CTA's channel block.
__device__ __forceinline__ void load_channels(const ScanArgs& p, int c0, float (&bias)[2], float* sskip) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int cb = c0 + warp * 8 + (lane & 3) * 2 + i;
    bias[i] = cb < p.C ? p.dt_b[cb] : 0.f;
  }
  if (threadIdx.x < kCh) sskip[threadIdx.x] = c0 + threadIdx.x < p.C ? p.d[c0 + threadIdx.x] : 0.f;
}

template <int NS, int TT>
__global__ void __launch_bounds__(kScanThreads) selective_scan_kernel(const ScanArgs p, const ScanSizes z) {
  extern __shared__ __align__(16) uint8_t ss_smem[];
  __shared__ __align__(16) float sskip[kCh];
  const int stage_bytes = scan_stage_bytes(z, TT);
  bf16* sw = reinterpret_cast<bf16*>(ss_smem + 2 * stage_bytes);
  float4* __restrict__ sdt = reinterpret_cast<float4*>(sw + kCh * z.cpitch);
  float* __restrict__ sy = reinterpret_cast<float*>(sdt + TT * kCh);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, q = lane & 3;
  const int c0 = blockIdx.x * kCh, cl = warp * 8 + (lane >> 2), c = c0 + cl;
  const bool in = c < p.C;
  const int4 seg = reinterpret_cast<const int4*>(p.segs)[blockIdx.y];  // {first row, rows, slot, position}
  pdl_wait();
  pdl_launch();
  load_wdt(p, z, c0, sw);
  float bias[2];
  load_channels(p, c0, bias, sskip);
  f32x2 A[NS / 2], S[NS / 2];
  float* st = p.state + (size_t)seg.z * p.state_pitch + (size_t)c * (4 * NS) + q * NS;
#pragma unroll
  for (int i = 0; i < NS / 2; ++i) {
    A[i] = in ? *reinterpret_cast<const f32x2*>(p.a + (size_t)c * (4 * NS) + q * NS + 2 * i) : 0ull;
    S[i] = in && seg.w > 0 ? *reinterpret_cast<const f32x2*>(st + 2 * i) : 0ull;
  }
  const int n_tiles = (seg.y + TT - 1) / TT;
  auto rows_of = [&](int j) { return seg.y - j * TT < TT ? seg.y - j * TT : TT; };
  load_tile<TT>(p, z, seg.x, rows_of(0), c0, Stage<TT>(ss_smem, z));
  cp_async_commit();
  for (int j = 0; j < n_tiles; ++j) {
    const Stage<TT> stage(ss_smem + (j & 1) * stage_bytes, z);
    if (j + 1 < n_tiles) load_tile<TT>(p, z, seg.x + (j + 1) * TT, rows_of(j + 1), c0, Stage<TT>(ss_smem + ((j + 1) & 1) * stage_bytes, z));
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const int n = rows_of(j);
    step_sizes<TT>(z, stage, sw, bias, n, sdt);
    __syncwarp();   // a warp computes the step sizes of its own channels
    const float* __restrict__ bc = stage.bc + q * (2 * NS);
    if constexpr (NS <= 8) {
      // Few warps are resident, so the instruction stream itself must offer parallel work: while a group of four tokens goes
      // through the recurrence, the next group's decays are computed and the one before is summed and stored.
      const float4* __restrict__ mine = sdt + cl;
      f32x2 decay[2][4][NS / 2], dx[2][4];
      float y[2][4];
      auto ahead = [&](int t0, int k) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const ulonglong2 dd = *reinterpret_cast<const ulonglong2*>(mine + (t0 + e) * kCh);
          dx[k][e] = dd.y;
          scan_decays<NS>(dd.x, A, decay[k][e]);
        }
      };
      ahead(0, 0);
#pragma unroll
      for (int g = 0; g < TT / 4; ++g) {
        if (g + 1 < TT / 4) ahead(4 * g + 4, (g + 1) & 1);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[g & 1][e] = scan_update<NS>(dx[g & 1][e], bc + (4 * g + e) * (8 * NS), decay[g & 1][e], S);
        if (g > 0) sy[(4 * g - 4 + q) * kYPitch + cl] = quad_transpose_sum(y[(g + 1) & 1], q);
      }
      sy[(TT - 4 + q) * kYPitch + cl] = quad_transpose_sum(y[(TT / 4 - 1) & 1], q);
    } else {
#pragma unroll 1
      for (int t0 = 0; t0 < TT; t0 += 4) {
        float y[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = scan_step<NS>(sdt + (t0 + e) * kCh + cl, bc + (t0 + e) * (8 * NS), A, S);
        sy[(t0 + q) * kYPitch + cl] = quad_transpose_sum(y, q);
      }
    }
    __syncthreads();
    store_tile<TT>(p, stage, sy, sskip, (size_t)seg.x + j * TT, n, c0, nullptr);
    __syncthreads();
  }
  if (in) {
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) *reinterpret_cast<f32x2*>(st + 2 * i) = S[i];
  }
}

// Decode: CTA = 32 channels of 16 slots; the states are requested before the projection that precedes the kernel is complete.
template <int NS>
__global__ void __launch_bounds__(kScanThreads) selective_scan_decode_kernel(const ScanArgs p, const ScanSizes z) {
  constexpr int kSlots = 16;
  constexpr int kAhead = NS <= 4 ? 16 : (NS == 8 ? 8 : 4);   // slots whose states are in registers at a time
  extern __shared__ __align__(16) uint8_t ss_smem[];
  __shared__ int s_pos[kSlots];
  __shared__ __align__(16) float sskip[kCh];
  const Stage<kSlots> stage(ss_smem, z);
  bf16* sw = reinterpret_cast<bf16*>(ss_smem + scan_stage_bytes(z, kSlots));
  float4* __restrict__ sdt = reinterpret_cast<float4*>(sw + kCh * z.cpitch);
  float* __restrict__ sy = reinterpret_cast<float*>(sdt + kSlots * kCh);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, q = lane & 3;
  const int c0 = blockIdx.x * kCh, cl = warp * 8 + (lane >> 2), c = c0 + cl;
  const bool in = c < p.C;
  const int b0 = blockIdx.y * kSlots;
  const int n = p.T - b0 < kSlots ? p.T - b0 : kSlots;
  if (threadIdx.x < kSlots) s_pos[threadIdx.x] = threadIdx.x < n ? p.seq_lens[b0 + threadIdx.x] - 1 : -1;
  load_wdt(p, z, c0, sw);
  float bias[2];
  load_channels(p, c0, bias, sskip);
  f32x2 A[NS / 2];
#pragma unroll
  for (int i = 0; i < NS / 2; ++i) A[i] = in ? *reinterpret_cast<const f32x2*>(p.a + (size_t)c * (4 * NS) + q * NS + 2 * i) : 0ull;
  __syncthreads();
  float* st = p.state + (size_t)b0 * p.state_pitch + (size_t)c * (4 * NS) + q * NS;
  f32x2 S[kAhead][NS / 2];
  auto request = [&](int s0) {
#pragma unroll
    for (int s = 0; s < kAhead; ++s)
#pragma unroll
      for (int i = 0; i < NS / 2; ++i)
        S[s][i] = in && s_pos[s0 + s] > 0 ? *reinterpret_cast<const f32x2*>(st + (size_t)(s0 + s) * p.state_pitch + 2 * i) : 0ull;
  };
  request(0);
  pdl_wait();
  pdl_launch();
  load_tile<kSlots>(p, z, b0, n, c0, stage);
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  step_sizes<kSlots>(z, stage, sw, bias, n, sdt);
  __syncwarp();
  const float* bc = stage.bc + q * (2 * NS);
#pragma unroll
  for (int s0 = 0; s0 < kSlots; s0 += kAhead) {
    if (s0 > 0) request(s0);
#pragma unroll
    for (int t0 = 0; t0 < kAhead; t0 += 4) {
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = s0 + t0 + e;
        y[e] = scan_step<NS>(sdt + t * kCh + cl, bc + t * (8 * NS), A, S[t0 + e]);
        if (in && s_pos[t] >= 0) {
#pragma unroll
          for (int i = 0; i < NS / 2; ++i) *reinterpret_cast<f32x2*>(st + (size_t)t * p.state_pitch + 2 * i) = S[t0 + e][i];
        }
      }
      sy[(s0 + t0 + q) * kYPitch + cl] = quad_transpose_sum(y, q);
    }
  }
  __syncthreads();
  store_tile<kSlots>(p, stage, sy, sskip, (size_t)b0, n, c0, s_pos);
}

template <int NS, int TT>
void launch_prompt(const ScanArgs& a, const ScanSizes& z, cudaStream_t s) {
  auto kernel = selective_scan_kernel<NS, TT>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, 220 * 1024, "selective_scan smem attr");
  AGRPO_PREFER_SMEM(kernel);
  launch_kernel(kernel, dim3((a.C + kCh - 1) / kCh, a.n_segs), dim3(kScanThreads), scan_smem_bytes(z, TT, 2), s, "selective_scan", a, z);
}

template <int NS>
bool launch_ns(const ScanArgs& a, cudaStream_t s) {
  const ScanSizes z = scan_sizes(a.rank, NS);
  if (a.segs != nullptr) {
    if (a.n_segs == 0) return true;
    if (scan_smem_bytes(z, 32, 2) <= 74 * 1024) launch_prompt<NS, 32>(a, z, s);
    else if (scan_smem_bytes(z, 16, 2) <= 220 * 1024) launch_prompt<NS, 16>(a, z, s);
    else return false;
    return true;
  }
  const int smem = scan_smem_bytes(z, 16, 1);
  if (smem > 220 * 1024) return false;
  if (a.T == 0) return true;
  auto kernel = selective_scan_decode_kernel<NS>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, 220 * 1024, "selective_scan_decode smem attr");
  AGRPO_PREFER_SMEM(kernel);
  launch_kernel(kernel, dim3((a.C + kCh - 1) / kCh, (a.T + 15) / 16), dim3(kScanThreads), smem, s, "selective_scan_decode", a, z);
  return true;
}

}  // namespace

int scan_code_pitch(int rank) { return (rank + 15) / 16 * 16 + 8; }   // rows of a fragment fall into different banks

int scan_states_per_lane(int N) { return N <= 8 ? 2 : N <= 16 ? 4 : N <= 32 ? 8 : N <= 64 ? 16 : 0; }

bool launch_selective_scan(const ScanArgs& a, cudaStream_t s) {
  switch (scan_states_per_lane(a.N)) {
    case 2: return launch_ns<2>(a, s);
    case 4: return launch_ns<4>(a, s);
    case 8: return launch_ns<8>(a, s);
    case 16: return launch_ns<16>(a, s);
    default: return false;
  }
}

bool selective_scan_serves(int N, int rank) {
  const int ns = scan_states_per_lane(N);
  return ns > 0 && scan_smem_bytes(scan_sizes(rank, ns), 16, 2) <= 220 * 1024;
}

}  // namespace agrpo
