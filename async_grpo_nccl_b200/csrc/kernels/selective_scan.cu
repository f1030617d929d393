// Selective scan (Mamba) in one kernel after the narrow projection of its input: step sizes on the tensor cores, softplus,
// decays, recurrence, read-out, skip and gate. The state lives in registers while a segment runs and in fp32 memory in between.
//
// Every (token, channel, state) needs one exponential, and the recurrence itself is sequential in time, so the kernel is laid
// out for the exponential units: four lanes share a channel, NS states each, 32 channels per CTA, and half of the warps do
// nothing but the recurrence, tile after tile, while the other half prepares the next tile and finishes the one before. Step
// sizes of a tile are a small matrix product with the channel block's rows of W_dt, done by mma.sync in place, so that they never
// exist in memory (they would be as large as the input in fp32). Read-outs of four tokens are summed over the four lanes at once:
// three shuffles, after which each lane holds one.
//
// The projection of the input arrives as the step-size code, bf16 rows of rank_p values (a multiple of 16) eight more apart, and
// B and C, fp32 [T, 8 NS]: for each quarter of the states NS values of B, then NS of C. Both are copied to shared memory as they
// are. A in log2 units [C, 4 NS]; state [slots, C, 4 NS].
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
constexpr int kMaxSmem = 220 * 1024;

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
// Buffers of a prompt CTA: while a tile goes through the recurrence, the next one's step sizes are computed and the one after
// that is loaded. A decode CTA has one of each.
struct ScanSmem {
  int code, bc, x, sdt, sy, sw, total;   // byte offsets
};
__host__ __device__ inline ScanSmem scan_smem(const ScanSizes& z, int tt, bool prompt) {
  ScanSmem m;
  const int two = prompt ? 2 : 1, three = prompt ? 3 : 1;
  m.code = 0;
  m.bc = m.code + two * tt * z.cpitch * 2;
  m.x = m.bc + three * tt * z.bc * 4;
  m.sdt = m.x + two * tt * kCh * 2;
  m.sy = m.sdt + two * tt * kCh * 8;
  m.sw = m.sy + two * tt * kYPitch * 4;
  m.total = m.sw + kCh * z.cpitch * 2;
  return m;
}

// The following run on 128 threads, `tid` of 128.
__device__ __forceinline__ void load_wdt(const ScanArgs& p, const ScanSizes& z, int c0, bf16* sw, int tid) {  // completes with the first tile
  for (int c = tid >> 5; c < kCh; c += 4)
    for (int k = (tid & 31) * 8; k < z.rank_p; k += 256) {
      if (c0 + c < p.C) cp_async16(sw + c * z.cpitch + k, reinterpret_cast<const bf16*>(p.wdt) + (size_t)(c0 + c) * p.ldw + k);
      else *reinterpret_cast<uint4*>(sw + c * z.cpitch + k) = make_uint4(0u, 0u, 0u, 0u);
    }
}

// Tile rows [0, n): code, B and C, x. Rows of the code, B and C from n on become zeros: their tokens are computed like the others,
// with a step size of zero, and must find finite numbers.
template <int TT>
__device__ __forceinline__ void load_tile(const ScanArgs& p, const ScanSizes& z, int row0, int n, int c0, bf16* scode, float* sbc, bf16* sx, int tid) {
  const uint8_t* code = reinterpret_cast<const uint8_t*>(p.code) + (size_t)row0 * z.cpitch * 2;
  const uint8_t* bc = reinterpret_cast<const uint8_t*>(p.r + (size_t)row0 * z.bc);
  const int n_code = n * z.cpitch / 8, n_bc = n * z.bc / 4;   // rows lie one after the other: flat copies of 16-byte pieces
  for (int i = tid; i < n_code; i += 128) cp_async16(reinterpret_cast<uint8_t*>(scode) + i * 16, code + (size_t)i * 16);
  for (int i = tid; i < n_bc; i += 128) cp_async16(reinterpret_cast<uint8_t*>(sbc) + i * 16, bc + (size_t)i * 16);
  if (n < TT) {
    for (int i = n_code + tid; i < TT * z.cpitch / 8; i += 128) reinterpret_cast<uint4*>(scode)[i] = make_uint4(0u, 0u, 0u, 0u);
    for (int i = n_bc + tid; i < TT * z.bc / 4; i += 128) reinterpret_cast<uint4*>(sbc)[i] = make_uint4(0u, 0u, 0u, 0u);
  }
  for (int i = tid; i < n * 4; i += 128) {
    const int t = i >> 2, k = (i & 3) * 8;
    if (c0 + k < p.C) cp_async16(sx + t * kCh + k, reinterpret_cast<const bf16*>(p.xc) + (size_t)(row0 + t) * p.ldx + c0 + k);
  }
}

// {dt, dt x} of TT tokens x 32 channels; tokens from n on get zeros, which leave a state as it is. Warp = 8 channels.
template <int TT>
__device__ __forceinline__ void step_sizes(const ScanSizes& z, const bf16* scode, const bf16* sx, const bf16* sw, const float (&bias)[2], int n,
                                           float2* sdt, int tid) {
  constexpr int M = TT / 16;
  const int warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, q2 = (lane & 3) * 2;
  float acc[M][4];
#pragma unroll
  for (int m = 0; m < M; ++m)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[m][e] = 0.f;
  const bf16* arow = scode + (lane & 15) * z.cpitch + (lane >> 4) * 8;
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
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      if (t < n) {
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sx + t * kCh + c));
        softplus_pair(acc[m][e] + bias[0], acc[m][e + 1] + bias[1], o.x, o.z);
        o.y = o.x * x.x;
        o.w = o.z * x.y;
      }
      *reinterpret_cast<float4*>(sdt + t * kCh + c) = o;
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
__device__ __forceinline__ float scan_step(const float2 d, const float* bc, const f32x2 (&A)[NS / 2], f32x2 (&S)[NS / 2]) {
  f32x2 e[NS / 2];
  scan_decays<NS>(pack2(d.x, d.x), A, e);
  return scan_update<NS>(pack2(d.y, d.y), bc, e, S);
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
__device__ __forceinline__ void store_tile(const ScanArgs& p, const float* sy, const float* sskip, size_t row0, int n, int c0, const int* s_pos, int tid) {
  for (int i = tid; i < n * 4; i += 128) {
    const int t = i >> 2, k = (i & 3) * 8;
    if (c0 + k >= p.C || (s_pos != nullptr && s_pos[t] < 0)) continue;
    float x[8], z[8], d[8], o[8];
    ld8(reinterpret_cast<const bf16*>(p.xc) + (row0 + t) * p.ldx + c0 + k, x);
    ld8(reinterpret_cast<const bf16*>(p.z) + (row0 + t) * p.ldz + c0 + k, z);
    ld8(sskip + k, d);
    ld8(sy + t * kYPitch + k, o);
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] = fmaf(d[e], x[e], o[e]) * z[e] * sigmoid_f32(z[e]);
    st8(reinterpret_cast<bf16*>(p.out) + (row0 + t) * p.ldo + c0 + k, o);
  }
}

// Constants of a CTA's channel block: step-size bias of the two columns that a thread holds of the small product, skip factors.
__device__ __forceinline__ void load_channels(const ScanArgs& p, int c0, float (&bias)[2], float* sskip, int tid) {
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int cb = c0 + (tid >> 5) * 8 + (tid & 3) * 2 + i;
    bias[i] = cb < p.C ? p.dt_b[cb] : 0.f;
  }
  if (tid < kCh) sskip[tid] = c0 + tid < p.C ? p.d[c0 + tid] : 0.f;
}

__device__ __forceinline__ void helper_bar() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

// Prompts: warps 0-3 do nothing but the recurrence, warps 4-7 everything around it (loads, step sizes, gate and store), a tile ahead
// and a tile behind.
template <int NS, int TT>
__global__ void __launch_bounds__(2 * kScanThreads) selective_scan_kernel(const ScanArgs p, const ScanSizes z) {
  extern __shared__ __align__(16) uint8_t ss_smem[];
  __shared__ __align__(16) float sskip[kCh];
  const ScanSmem off = scan_smem(z, TT, true);
  bf16* scode = reinterpret_cast<bf16*>(ss_smem + off.code);
  float* sbc = reinterpret_cast<float*>(ss_smem + off.bc);
  bf16* sx = reinterpret_cast<bf16*>(ss_smem + off.x);
  float2* __restrict__ sdt = reinterpret_cast<float2*>(ss_smem + off.sdt);
  float* __restrict__ sy = reinterpret_cast<float*>(ss_smem + off.sy);
  bf16* sw = reinterpret_cast<bf16*>(ss_smem + off.sw);
  const bool helper = threadIdx.x >= kScanThreads;
  const int tid = threadIdx.x & (kScanThreads - 1);
  const int c0 = blockIdx.x * kCh;
  const int4 seg = reinterpret_cast<const int4*>(p.segs)[blockIdx.y];  // {first row, rows, slot, position}
  const int n_tiles = (seg.y + TT - 1) / TT;
  auto rows_of = [&](int j) { return seg.y - j * TT < TT ? seg.y - j * TT : TT; };
  pdl_wait();
  pdl_launch();
  if (helper) {
    auto load = [&](int j) {
      if (j < n_tiles)
        load_tile<TT>(p, z, seg.x + j * TT, rows_of(j), c0, scode + (j & 1) * TT * z.cpitch, sbc + (j % 3) * TT * (8 * NS), sx + (j & 1) * TT * kCh, tid);
      cp_async_commit();
    };
    float bias[2];
    auto sizes = [&](int j) {  // the tile's load is complete for this thread
      helper_bar();
      step_sizes<TT>(z, scode + (j & 1) * TT * z.cpitch, sx + (j & 1) * TT * kCh, sw, bias, rows_of(j), sdt + (j & 1) * TT * kCh, tid);
    };
    load_wdt(p, z, c0, sw, tid);
    load(0);
    load(1);
    load_channels(p, c0, bias, sskip, tid);
    cp_async_wait<1>();
    sizes(0);
    __syncthreads();
    for (int j = 0; j < n_tiles; ++j) {
      load(j + 2);
      if (j + 1 < n_tiles) {
        cp_async_wait<1>();
        sizes(j + 1);
      }
      if (j > 0) store_tile(p, sy + ((j - 1) & 1) * TT * kYPitch, sskip, (size_t)seg.x + (j - 1) * TT, TT, c0, nullptr, tid);
      cp_async_wait<1>();   // B and C of the next tile, also where no step sizes were due
      __syncthreads();
    }
    store_tile(p, sy + ((n_tiles - 1) & 1) * TT * kYPitch, sskip, (size_t)seg.x + (n_tiles - 1) * TT, rows_of(n_tiles - 1), c0, nullptr, tid);
    return;
  }
  const int lane = tid & 31, q = lane & 3;
  const int cl = (tid >> 5) * 8 + (lane >> 2), c = c0 + cl;
  const bool in = c < p.C;
  f32x2 A[NS / 2], S[NS / 2];
  float* st = p.state + (size_t)seg.z * p.state_pitch + (size_t)c * (4 * NS) + q * NS;
#pragma unroll
  for (int i = 0; i < NS / 2; ++i) {
    A[i] = in ? *reinterpret_cast<const f32x2*>(p.a + (size_t)c * (4 * NS) + q * NS + 2 * i) : 0ull;
    S[i] = in && seg.w > 0 ? *reinterpret_cast<const f32x2*>(st + 2 * i) : 0ull;
  }
  __syncthreads();
  for (int j = 0; j < n_tiles; ++j) {
    const float2* __restrict__ mine = sdt + (j & 1) * TT * kCh + cl;
    const float* __restrict__ bc = sbc + (j % 3) * TT * (8 * NS) + q * (2 * NS);
    float* __restrict__ ys = sy + ((j & 1) * TT + q) * kYPitch + cl;
    if constexpr (NS <= 8) {
      // Few warps are resident, so the instruction stream itself must offer parallel work: while a group of four tokens goes
      // through the recurrence, the next group's decays are computed and the one before is summed and stored.
      f32x2 decay[2][4][NS / 2];
      float dx[2][4], y[2][4];
      auto ahead = [&](int t0, int k) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 d = mine[(t0 + e) * kCh];
          dx[k][e] = d.y;
          scan_decays<NS>(pack2(d.x, d.x), A, decay[k][e]);
        }
      };
      ahead(0, 0);
#pragma unroll
      for (int g = 0; g < TT / 4; ++g) {
        if (g + 1 < TT / 4) ahead(4 * g + 4, (g + 1) & 1);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[g & 1][e] = scan_update<NS>(pack2(dx[g & 1][e], dx[g & 1][e]), bc + (4 * g + e) * (8 * NS), decay[g & 1][e], S);
        if (g > 0) ys[(4 * g - 4) * kYPitch] = quad_transpose_sum(y[(g + 1) & 1], q);
      }
      ys[(TT - 4) * kYPitch] = quad_transpose_sum(y[(TT / 4 - 1) & 1], q);
    } else {
#pragma unroll 1
      for (int t0 = 0; t0 < TT; t0 += 4) {
        float y[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = scan_step<NS>(mine[(t0 + e) * kCh], bc + (t0 + e) * (8 * NS), A, S);
        ys[t0 * kYPitch] = quad_transpose_sum(y, q);
      }
    }
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
  const ScanSmem off = scan_smem(z, kSlots, false);
  bf16* scode = reinterpret_cast<bf16*>(ss_smem + off.code);
  float* sbc = reinterpret_cast<float*>(ss_smem + off.bc);
  bf16* sx = reinterpret_cast<bf16*>(ss_smem + off.x);
  float2* __restrict__ sdt = reinterpret_cast<float2*>(ss_smem + off.sdt);
  float* __restrict__ sy = reinterpret_cast<float*>(ss_smem + off.sy);
  bf16* sw = reinterpret_cast<bf16*>(ss_smem + off.sw);
  const int tid = threadIdx.x, lane = tid & 31, q = lane & 3;
  const int c0 = blockIdx.x * kCh, cl = (tid >> 5) * 8 + (lane >> 2), c = c0 + cl;
  const bool in = c < p.C;
  const int b0 = blockIdx.y * kSlots;
  const int n = p.T - b0 < kSlots ? p.T - b0 : kSlots;
  if (tid < kSlots) s_pos[tid] = tid < n ? p.seq_lens[b0 + tid] - 1 : -1;
  load_wdt(p, z, c0, sw, tid);
  float bias[2];
  load_channels(p, c0, bias, sskip, tid);
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
  load_tile<kSlots>(p, z, b0, n, c0, scode, sbc, sx, tid);
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  step_sizes<kSlots>(z, scode, sx, sw, bias, n, sdt, tid);
  __syncwarp();   // a warp computes the step sizes of its own channels
  const float* bc = sbc + q * (2 * NS);
#pragma unroll
  for (int s0 = 0; s0 < kSlots; s0 += kAhead) {
    if (s0 > 0) request(s0);
#pragma unroll
    for (int t0 = 0; t0 < kAhead; t0 += 4) {
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = s0 + t0 + e;
        y[e] = scan_step<NS>(sdt[t * kCh + cl], bc + t * (8 * NS), A, S[t0 + e]);
        if (in && s_pos[t] >= 0) {
#pragma unroll
          for (int i = 0; i < NS / 2; ++i) *reinterpret_cast<f32x2*>(st + (size_t)t * p.state_pitch + 2 * i) = S[t0 + e][i];
        }
      }
      sy[(s0 + t0 + q) * kYPitch + cl] = quad_transpose_sum(y, q);
    }
  }
  __syncthreads();
  store_tile(p, sy, sskip, (size_t)b0, n, c0, s_pos, tid);
}

template <int NS, int TT>
void launch_prompt(const ScanArgs& a, const ScanSizes& z, cudaStream_t s) {
  auto kernel = selective_scan_kernel<NS, TT>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, kMaxSmem, "selective_scan smem attr");
  AGRPO_PREFER_SMEM(kernel);
  launch_kernel(kernel, dim3((a.C + kCh - 1) / kCh, a.n_segs), dim3(2 * kScanThreads), scan_smem(z, TT, true).total, s, "selective_scan", a, z);
}

template <int NS>
bool launch_ns(const ScanArgs& a, cudaStream_t s) {
  const ScanSizes z = scan_sizes(a.rank, NS);
  if (a.segs != nullptr) {
    if (scan_smem(z, 16, true).total > kMaxSmem) return false;
    if (a.n_segs == 0) return true;
    if (scan_smem(z, 32, true).total <= 74 * 1024) launch_prompt<NS, 32>(a, z, s);   // three CTAs to an SM
    else launch_prompt<NS, 16>(a, z, s);
    return true;
  }
  const int smem = scan_smem(z, 16, false).total;
  if (smem > kMaxSmem) return false;
  if (a.T == 0) return true;
  auto kernel = selective_scan_decode_kernel<NS>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, kMaxSmem, "selective_scan_decode smem attr");
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
  return ns > 0 && scan_smem(scan_sizes(rank, ns), 16, true).total <= kMaxSmem;
}

}  // namespace agrpo
