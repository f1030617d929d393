// Selective scan (Mamba) in one kernel after the narrow projection of its input: step sizes on the tensor cores, softplus,
// decays, recurrence, read-out, skip and gate. The state lives in registers while a segment runs and in fp32 memory in between.
//
// Every (token, channel, state) needs one exponential, and the recurrence itself is sequential in time, so the kernel is laid
// out for the exponential units: four lanes share a channel, NS states each, 32 channels per CTA, and a segment's tokens go
// through shared memory in tiles that are loaded one ahead. Step sizes of a tile are a small matrix product with the channel
// block's rows of W_dt, done by mma.sync in place, so that they never exist in memory (they would be as large as the input in
// fp32). Read-outs of four tokens are summed over the four lanes at once: three shuffles, after which each lane finishes one.
//
// Layout of r [T, ldr] fp32: step-size code (rank_p columns, a multiple of 16), then for each quarter q of the states NS values
// of B and NS values of C. A in log2 units, [C, 4 NS]; state [slots, C, 4 NS].
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
// where the odd series converges by 1/9 a term (the first one left out is below 1e-9 of the sum).
__device__ __forceinline__ float softplus_f32(float v) {
  const float e = __expf(-fabsf(v));
  const float s = __fdividef(e, 2.f + e);
  const float q = s * s;
  float p = 1.f / 17.f;
  p = fmaf(p, q, 1.f / 15.f);
  p = fmaf(p, q, 1.f / 13.f);
  p = fmaf(p, q, 1.f / 11.f);
  p = fmaf(p, q, 1.f / 9.f);
  p = fmaf(p, q, 1.f / 7.f);
  p = fmaf(p, q, 1.f / 5.f);
  p = fmaf(p, q, 1.f / 3.f);
  p = fmaf(p, q, 1.f);
  return fmaxf(v, 0.f) + 2.f * s * p;
}

struct ScanSizes {
  int rank_p, wpitch, rpitch;   // bf16 elements / floats per row in shared memory
  int r_floats;                 // columns of r
};
__host__ __device__ inline ScanSizes scan_sizes(int rank, int ns) {
  ScanSizes z;
  z.rank_p = (rank + 15) / 16 * 16;
  z.r_floats = z.rank_p + 8 * ns;
  z.wpitch = z.rank_p + 8;
  z.rpitch = z.r_floats;
  while (z.rpitch % 32 != 8) z.rpitch += 4;   // rows of a fragment fall into different banks
  return z;
}
// stage: r tile, x tile, z tile; then W_dt rows, {dt, dt x} pairs
__host__ __device__ inline int scan_stage_bytes(const ScanSizes& z, int tt) { return tt * z.rpitch * 4 + 2 * tt * kCh * 2; }
inline int scan_smem_bytes(const ScanSizes& z, int tt, int stages) {
  return stages * scan_stage_bytes(z, tt) + kCh * z.wpitch * 2 + tt * kCh * 8;
}

__device__ __forceinline__ void load_wdt(const ScanArgs& p, const ScanSizes& z, int c0, bf16* sw) {
  const int per = z.rank_p / 8;
  for (int i = threadIdx.x; i < kCh * per; i += kScanThreads) {
    const int c = i / per, k = (i % per) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (c0 + c < p.C) v = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(p.wdt) + (size_t)(c0 + c) * p.ldw + k);
    *reinterpret_cast<uint4*>(sw + c * z.wpitch + k) = v;
  }
}

// Tile rows [0, n) of r, x and z into a stage; x and z rows are kCh channels. Rows of r from n on become zeros: their tokens are
// computed like the others, with a step size of zero, and must find finite numbers.
template <int TT>
__device__ __forceinline__ void load_tile(const ScanArgs& p, const ScanSizes& z, int row0, int n, int c0, uint8_t* stage) {
  const int per = z.r_floats / 4;
  for (int i = threadIdx.x; i < n * per; i += kScanThreads) {
    const int t = i / per, k = (i % per) * 4;
    cp_async16(stage + (t * z.rpitch + k) * 4, p.r + (size_t)(row0 + t) * p.ldr + k);
  }
  for (int i = n * per + threadIdx.x; i < TT * per; i += kScanThreads)
    *reinterpret_cast<float4*>(stage + ((i / per) * z.rpitch + (i % per) * 4) * 4) = make_float4(0.f, 0.f, 0.f, 0.f);
  uint8_t* sx = stage + TT * z.rpitch * 4;
  uint8_t* sz = sx + TT * kCh * 2;
  for (int i = threadIdx.x; i < n * 4; i += kScanThreads) {
    const int t = i >> 2, k = (i & 3) * 8;
    if (c0 + k < p.C) {
      cp_async16(sx + (t * kCh + k) * 2, reinterpret_cast<const bf16*>(p.xc) + (size_t)(row0 + t) * p.ldx + c0 + k);
      cp_async16(sz + (t * kCh + k) * 2, reinterpret_cast<const bf16*>(p.z) + (size_t)(row0 + t) * p.ldz + c0 + k);
    }
  }
}

// {dt, dt x} of TT tokens x 32 channels; tokens from n on get zeros, which leave a state as it is. Warp = 8 channels.
template <int TT>
__device__ __forceinline__ void step_sizes(const ScanSizes& z, const float* sr, const bf16* sx, const bf16* sw, const float (&bias)[2], int n, float2* sdt) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, q2 = (lane & 3) * 2;
  const bf16* wrow = sw + (warp * 8 + g) * z.wpitch;
#pragma unroll
  for (int m = 0; m < TT / 16; ++m) {
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const float* r0 = sr + (m * 16 + g) * z.rpitch;
    const float* r1 = r0 + 8 * z.rpitch;
    for (int k = 0; k < z.rank_p; k += 16) {
      const float2 a0 = *reinterpret_cast<const float2*>(r0 + k + q2), a1 = *reinterpret_cast<const float2*>(r1 + k + q2);
      const float2 a2 = *reinterpret_cast<const float2*>(r0 + k + q2 + 8), a3 = *reinterpret_cast<const float2*>(r1 + k + q2 + 8);
      mma_16816(acc, pack_bf16x2(a0.x, a0.y), pack_bf16x2(a1.x, a1.y), pack_bf16x2(a2.x, a2.y), pack_bf16x2(a3.x, a3.y),
                *reinterpret_cast<const uint32_t*>(wrow + k + q2), *reinterpret_cast<const uint32_t*>(wrow + k + q2 + 8));
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = m * 16 + g + (e >> 1) * 8, c = warp * 8 + q2 + (e & 1);
      float2 o = make_float2(0.f, 0.f);
      if (t < n) {
        o.x = softplus_f32(acc[e] + bias[e & 1]);
        o.y = o.x * __bfloat162float(sx[t * kCh + c]);
      }
      sdt[t * kCh + c] = o;
    }
  }
}

// One token of one channel quarter: S <- exp2(dt A) S + (dt x) B, returns this quarter's part of S . C.
template <int NS>
__device__ __forceinline__ float scan_step(const float2 d, const float* bc, const f32x2 (&A)[NS / 2], f32x2 (&S)[NS / 2]) {
  const f32x2 dt = pack2(d.x, d.x), dx = pack2(d.y, d.y);
  f32x2 y = 0;  // bits of {0.f, 0.f}
#pragma unroll
  for (int i = 0; i < NS / 2; ++i) {
    float a, b;
    unpack2(mul2(dt, A[i]), a, b);
    const f32x2 B = *reinterpret_cast<const f32x2*>(bc + 2 * i), C = *reinterpret_cast<const f32x2*>(bc + NS + 2 * i);
    S[i] = fma2(pack2(ex2(a), ex2(b)), S[i], mul2(dx, B));
    y = fma2(S[i], C, y);
  }
  float a, b;
  unpack2(y, a, b);
  return a + b;
}

// Sums over the four lanes of a channel for four tokens: lane q gets token q.
__device__ __forceinline__ float quad_transpose_sum(const float (&y)[4], int q) {
  const bool odd = q & 1, high = q & 2;
  float a = odd ? y[1] : y[0], b = odd ? y[3] : y[2];
  a += __shfl_xor_sync(0xffffffffu, odd ? y[0] : y[1], 1);
  b += __shfl_xor_sync(0xffffffffu, odd ? y[2] : y[3], 1);
  return (high ? b : a) + __shfl_xor_sync(0xffffffffu, high ? a : b, 2);
}

template <int NS, int TT>
__global__ void __launch_bounds__(kScanThreads) selective_scan_kernel(const ScanArgs p, const ScanSizes z) {
  extern __shared__ __align__(16) uint8_t ss_smem[];
  const int stage_bytes = scan_stage_bytes(z, TT);
  bf16* sw = reinterpret_cast<bf16*>(ss_smem + 2 * stage_bytes);
  float2* sdt = reinterpret_cast<float2*>(reinterpret_cast<uint8_t*>(sw) + kCh * z.wpitch * 2);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, q = lane & 3;
  const int c0 = blockIdx.x * kCh, cl = warp * 8 + (lane >> 2), c = c0 + cl;
  const bool in = c < p.C;
  const int4 seg = reinterpret_cast<const int4*>(p.segs)[blockIdx.y];  // {first row, rows, slot, position}
  pdl_wait();
  pdl_launch();
  load_wdt(p, z, c0, sw);
  float bias[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int cb = c0 + warp * 8 + (lane & 3) * 2 + i;
    bias[i] = cb < p.C ? p.dt_b[cb] : 0.f;
  }
  const float skip = in ? p.d[c] : 0.f;
  f32x2 A[NS / 2], S[NS / 2];
  float* st = p.state + (size_t)seg.z * p.state_pitch + (size_t)c * (4 * NS) + q * NS;
#pragma unroll
  for (int i = 0; i < NS / 2; ++i) {
    A[i] = in ? *reinterpret_cast<const f32x2*>(p.a + (size_t)c * (4 * NS) + q * NS + 2 * i) : 0ull;
    S[i] = in && seg.w > 0 ? *reinterpret_cast<const f32x2*>(st + 2 * i) : 0ull;
  }
  const int n_tiles = (seg.y + TT - 1) / TT;
  auto rows_of = [&](int j) { return seg.y - j * TT < TT ? seg.y - j * TT : TT; };
  load_tile<TT>(p, z, seg.x, rows_of(0), c0, ss_smem);
  cp_async_commit();
  for (int j = 0; j < n_tiles; ++j) {
    uint8_t* stage = ss_smem + (j & 1) * stage_bytes;
    if (j + 1 < n_tiles) load_tile<TT>(p, z, seg.x + (j + 1) * TT, rows_of(j + 1), c0, ss_smem + ((j + 1) & 1) * stage_bytes);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const float* sr = reinterpret_cast<const float*>(stage);
    bf16* sx = reinterpret_cast<bf16*>(stage + TT * z.rpitch * 4);
    const bf16* sz = sx + TT * kCh;
    const int n = rows_of(j);
    step_sizes<TT>(z, sr, sx, sw, bias, n, sdt);
    __syncwarp();   // a warp computes the step sizes of its own channels
    const float* bc = sr + z.rank_p + q * (2 * NS);
#pragma unroll 2
    for (int t0 = 0; t0 < TT; t0 += 4) {
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = scan_step<NS>(sdt[(t0 + e) * kCh + cl], bc + (t0 + e) * z.rpitch, A, S);
      float v = quad_transpose_sum(y, q);
      const int t = t0 + q;
      const float x = __bfloat162float(sx[t * kCh + cl]), g = __bfloat162float(sz[t * kCh + cl]);
      v = fmaf(skip, x, v);
      sx[t * kCh + cl] = __float2bfloat16(v * g * sigmoid_f32(g));  // read for the last time: the result takes its place
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * 4; i += kScanThreads) {
      const int t = i >> 2, k = (i & 3) * 8;
      if (c0 + k < p.C)
        *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.out) + (size_t)(seg.x + j * TT + t) * p.ldo + c0 + k) =
            *reinterpret_cast<const uint4*>(sx + t * kCh + k);
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
  const int stage_bytes = scan_stage_bytes(z, kSlots);
  bf16* sw = reinterpret_cast<bf16*>(ss_smem + stage_bytes);
  float2* sdt = reinterpret_cast<float2*>(reinterpret_cast<uint8_t*>(sw) + kCh * z.wpitch * 2);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, q = lane & 3;
  const int c0 = blockIdx.x * kCh, cl = warp * 8 + (lane >> 2), c = c0 + cl;
  const bool in = c < p.C;
  const int b0 = blockIdx.y * kSlots;
  const int n = p.T - b0 < kSlots ? p.T - b0 : kSlots;
  load_wdt(p, z, c0, sw);
  if (threadIdx.x < kSlots) s_pos[threadIdx.x] = threadIdx.x < n ? p.seq_lens[b0 + threadIdx.x] - 1 : -1;
  float bias[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int cb = c0 + warp * 8 + (lane & 3) * 2 + i;
    bias[i] = cb < p.C ? p.dt_b[cb] : 0.f;
  }
  const float skip = in ? p.d[c] : 0.f;
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
  load_tile<kSlots>(p, z, b0, n, c0, ss_smem);
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  const float* sr = reinterpret_cast<const float*>(ss_smem);
  bf16* sx = reinterpret_cast<bf16*>(ss_smem + kSlots * z.rpitch * 4);
  const bf16* sz = sx + kSlots * kCh;
  step_sizes<kSlots>(z, sr, sx, sw, bias, n, sdt);
  __syncwarp();
  const float* bc = sr + z.rank_p + q * (2 * NS);
#pragma unroll
  for (int s0 = 0; s0 < kSlots; s0 += kAhead) {
    if (s0 > 0) request(s0);
#pragma unroll
    for (int t0 = 0; t0 < kAhead; t0 += 4) {
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = s0 + t0 + e;
        y[e] = scan_step<NS>(sdt[t * kCh + cl], bc + t * z.rpitch, A, S[t0 + e]);
        if (in && s_pos[t] >= 0) {
#pragma unroll
          for (int i = 0; i < NS / 2; ++i) *reinterpret_cast<f32x2*>(st + (size_t)t * p.state_pitch + 2 * i) = S[t0 + e][i];
        }
      }
      float v = quad_transpose_sum(y, q);
      const int t = s0 + t0 + q;
      const float x = __bfloat162float(sx[t * kCh + cl]), g = __bfloat162float(sz[t * kCh + cl]);
      v = fmaf(skip, x, v);
      sx[t * kCh + cl] = __float2bfloat16(v * g * sigmoid_f32(g));
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < n * 4; i += kScanThreads) {
    const int t = i >> 2, k = (i & 3) * 8;
    if (c0 + k < p.C && s_pos[t] >= 0)
      *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.out) + (size_t)(b0 + t) * p.ldo + c0 + k) = *reinterpret_cast<const uint4*>(sx + t * kCh + k);
  }
}

template <int NS, int TT>
void launch_prompt(const ScanArgs& a, const ScanSizes& z, cudaStream_t s) {
  auto kernel = selective_scan_kernel<NS, TT>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, 220 * 1024, "selective_scan smem attr");
  launch_kernel(kernel, dim3((a.C + kCh - 1) / kCh, a.n_segs), dim3(kScanThreads), scan_smem_bytes(z, TT, 2), s, "selective_scan", a, z);
}

template <int NS>
bool launch_ns(const ScanArgs& a, cudaStream_t s) {
  const ScanSizes z = scan_sizes(a.rank, NS);
  if (a.segs != nullptr) {
    if (a.n_segs == 0) return true;
    if (scan_smem_bytes(z, 32, 2) <= 72 * 1024) launch_prompt<NS, 32>(a, z, s);
    else if (scan_smem_bytes(z, 16, 2) <= 220 * 1024) launch_prompt<NS, 16>(a, z, s);
    else return false;
    return true;
  }
  const int smem = scan_smem_bytes(z, 16, 1);
  if (smem > 220 * 1024) return false;
  if (a.T == 0) return true;
  auto kernel = selective_scan_decode_kernel<NS>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, 220 * 1024, "selective_scan_decode smem attr");
  launch_kernel(kernel, dim3((a.C + kCh - 1) / kCh, (a.T + 15) / 16), dim3(kScanThreads), smem, s, "selective_scan_decode", a, z);
  return true;
}

}  // namespace

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
