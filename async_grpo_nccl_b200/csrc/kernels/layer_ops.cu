// Listed-layer operations in their plain form, for bf16 and for 32-bit activations: embedding + first norm, short
// convolution with its per-sequence ring, sliding-window attention with mixed heads (any head size), true fp32 GEMMs with
// the same fused epilogues as the tensor-core ones, and sampling from fp32 logits. Built without fast-math.
#include "../common/ptx.cuh"
#include "../launchers.h"
#include "../launchers_layers.h"
#include "layer_ops.cuh"

namespace agrpo {

namespace {

typedef __nv_bfloat16 bf16;

template <typename T>
DytNorm<T> as_norm(const DytArgs& n) {
  return DytNorm<T>{reinterpret_cast<const T*>(n.w), reinterpret_cast<const T*>(n.b), reinterpret_cast<const T*>(n.alpha)};
}

// ------------------------------------------------------------------------------------------------
template <typename T>
__global__ void embed_dyt_kernel(const int* __restrict__ ids, const T* __restrict__ table, float scale, float* __restrict__ x,
                                 T* __restrict__ h, DytNorm<T> n, int T_, int W, int V) {
  pdl_wait();
  pdl_launch();
  const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (row >= T_) return;
  int id = ids[row];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  const float a = ldf(n.alpha);
  for (int c = (threadIdx.x & 31) * 8; c < W; c += 256) {
    float e[8], w[8], b[8], y[8];
    ld8(table + (size_t)id * W + c, e);
    ld8(n.w + c, w);
    ld8(n.b + c, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      e[i] *= scale;
      y[i] = fmaf(tanh_f32(a * e[i]), w[i], b[i]);
    }
    st8(x + (size_t)row * W + c, e);
    st8(h + (size_t)row * W + c, y);
  }
}

// ------------------------------------------------------------------------------------------------
// Short convolution. Thread = 8 channels of kConvRows consecutive token rows. Inside a segment the rows it needs are loaded
// up front and stay in registers; a tile at a segment's start, or with rows of several segments, goes row by row and takes
// older values from the ring.
constexpr int kConvRows = 8;

template <typename T>
struct ConvVec;
template <>
struct ConvVec<bf16> {
  uint4 v;
  __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ float get(int i) const {
    const uint32_t w = i < 2 ? v.x : (i < 4 ? v.y : (i < 6 ? v.z : v.w));
    return __uint_as_float((i & 1) ? (w & 0xffff0000u) : (w << 16));
  }
};
template <>
struct ConvVec<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) {
    a = *reinterpret_cast<const float4*>(p);
    b = *reinterpret_cast<const float4*>(p + 4);
  }
  __device__ __forceinline__ float get(int i) const {
    return i == 0 ? a.x : i == 1 ? a.y : i == 2 ? a.z : i == 3 ? a.w : i == 4 ? b.x : i == 5 ? b.y : i == 6 ? b.z : b.w;
  }
};

template <typename T>
__device__ __forceinline__ void conv_store(const ShortConvArgs& p, int t, const int4& r, int c, float (&acc)[8]) {
  if (p.bias != nullptr) {
    float b[8];
    ld8(reinterpret_cast<const T*>(p.bias) + c, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] += b[i];
  }
  if (p.silu) {
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = sizeof(T) == 4 ? acc[i] / (1.f + expf(-acc[i])) : acc[i] * sigmoid_f32(acc[i]);
  }
  if (c < p.q_cols) {
    st8(reinterpret_cast<T*>(p.q_out) + (size_t)t * p.q_cols + c, acc);
    return;
  }
  const int blk = p.block_tables[(size_t)r.x * p.max_blocks + r.y / p.block_size];
  if (blk < 0 || blk >= p.num_cache_blocks) {
    report_status(p.status, kStatusBadIndex);
    return;
  }
  const int kc = c - p.q_cols, g = kc / p.D, d = kc % p.D, G = p.k_cols / p.D;
  st8(reinterpret_cast<T*>(p.k_cache) + (((size_t)blk * G + g) * p.block_size + r.y % p.block_size) * p.D + d, acc);
}

template <typename T>
__device__ __forceinline__ void conv_row(const ShortConvArgs& p, const RowMap& map, int t, int c, int C) {
  const int4 r = map.get(t);
  if (r.y < 0) return;
  const T* u = reinterpret_cast<const T*>(p.u);
  const T* ring = reinterpret_cast<const T*>(p.ring);
  const T* w = reinterpret_cast<const T*>(p.w) + c;
  float acc[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.f;
  for (int back = p.taps - 1; back >= 0; --back) {  // oldest first
    if (r.y - back < 0) continue;
    const int row = t - back;
    const T* src = row >= r.z ? u + (size_t)row * p.ldu + c
                              : ring + (size_t)r.x * p.ring_pitch + (size_t)((r.y - back) % p.ring_len) * C + c;
    float v[8], x[8];
    ld8(src, v);
    ld8(w + (size_t)(p.taps - 1 - back) * C, x);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = fmaf(x[i], v[i], acc[i]);
  }
  conv_store<T>(p, t, r, c, acc);
}

// TAPS = 0: any number of taps, row by row
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) short_conv_kernel(ShortConvArgs p) {
  pdl_wait();
  pdl_launch();
  const int C = p.q_cols + p.k_cols;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (c >= C) return;
  const RowMap map{reinterpret_cast<const int4*>(p.rows), p.seq_lens};
  const int t0 = blockIdx.x * kConvRows;
  const int n = p.T - t0 < kConvRows ? p.T - t0 : kConvRows;
  if constexpr (TAPS > 0) {
    if (p.rows != nullptr && n == kConvRows) {
      const int4 first = map.get(t0), last = map.get(t0 + kConvRows - 1);
      if (first.z == last.z && t0 - (TAPS - 1) >= first.z) {
        const T* u = reinterpret_cast<const T*>(p.u) + c;
        ConvVec<T> v[kConvRows + TAPS - 1];
#pragma unroll
        for (int i = 0; i < kConvRows + TAPS - 1; ++i) v[i].load(u + (size_t)(t0 - (TAPS - 1) + i) * p.ldu);
        float w[TAPS][8];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) ld8(reinterpret_cast<const T*>(p.w) + (size_t)k * C + c, w[k]);
#pragma unroll
        for (int r = 0; r < kConvRows; ++r) {
          float acc[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            acc[i] = 0.f;
#pragma unroll
            for (int k = 0; k < TAPS; ++k) acc[i] = fmaf(w[k][i], v[r + k].get(i), acc[i]);
          }
          conv_store<T>(p, t0 + r, make_int4(first.x, first.y + r, first.z, 0), c, acc);
        }
        return;
      }
    }
  }
  for (int r = 0; r < n; ++r) conv_row<T>(p, map, t0 + r, c, C);
}

// Decode rows (row = slot), thread = 8 channels of one row: convolution and ring in one pass. The ring has room for `taps` values,
// so the new one takes the place of one that no tap reads any more.
template <typename T>
__global__ void __launch_bounds__(128) short_conv_decode_kernel(ShortConvArgs p) {
  pdl_wait();
  pdl_launch();
  const int C = p.q_cols + p.k_cols;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8, t = blockIdx.x;
  const int pos = p.seq_lens[t] - 1;
  if (c >= C || pos < 0) return;
  const T* w = reinterpret_cast<const T*>(p.w) + c;
  T* ring = reinterpret_cast<T*>(p.ring) + (size_t)t * p.ring_pitch + c;
  float v[8], acc[8], x[8];
  ld8(reinterpret_cast<const T*>(p.u) + (size_t)t * p.ldu + c, v);
  ld8(w + (size_t)(p.taps - 1) * C, x);
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.f;
#pragma unroll 4
  for (int back = p.taps - 1; back > 0; --back) {  // oldest first
    if (pos - back < 0) continue;
    float y[8], xw[8];
    ld8(ring + (size_t)((pos - back) % p.ring_len) * C, y);
    ld8(w + (size_t)(p.taps - 1 - back) * C, xw);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = fmaf(xw[i], y[i], acc[i]);
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = fmaf(x[i], v[i], acc[i]);
  if (p.taps > 1) st8(ring + (size_t)(pos % p.ring_len) * C, v);
  conv_store<T>(p, t, make_int4(t, pos, t, 0), c, acc);
}

// ring_rows: the rows whose values later steps need (the last ring_len of each segment); decode: every row
template <typename T>
__global__ void short_conv_ring_kernel(ShortConvArgs p, const int* __restrict__ ring_rows) {
  pdl_wait();
  pdl_launch();
  const int C = p.q_cols + p.k_cols;
  const int t = ring_rows != nullptr ? ring_rows[blockIdx.x] : blockIdx.x;
  if (t < 0 || t >= p.T) return;
  const RowMap map{reinterpret_cast<const int4*>(p.rows), p.seq_lens};
  const int4 r = map.get(t);
  if (r.y < 0) return;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (c >= C) return;
  float v[8];
  ld8(reinterpret_cast<const T*>(p.u) + (size_t)t * p.ldu + c, v);
  st8(reinterpret_cast<T*>(p.ring) + (size_t)r.x * p.ring_pitch + (size_t)(r.y % p.ring_len) * C + c, v);
}

// ------------------------------------------------------------------------------------------------
// Sliding-window attention, one CTA per token row, all heads. Pass 1 over the visible keys gives every head's maximum
// and sum; pass 2 recomputes the scores, turns them into final softmax weights, mixes them across heads and
// accumulates the values. Keys are staged one key head at a time. Works for any head size; the tensor-core kernels
// replace it where they apply.
constexpr int kWaKeys = 32;
constexpr int kWaThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kWaThreads) window_attn_kernel(WindowAttnArgs p) {
  pdl_wait();
  pdl_launch();
  extern __shared__ float wa_smem[];
  const int H = p.H, G = p.G, D = p.D, grp = H / G;
  const int kp = D + 1;                       // padded key pitch
  float* sq = wa_smem;                        // [H, D]
  float* sacc = sq + H * D;                   // [H, D]
  float* sk = sacc + H * D;                   // [keys, kp]
  float* sw = sk + kWaKeys * kp;              // [H, keys + 1]
  float* smix = sw + H * (kWaKeys + 1);       // [H, keys + 1]
  float* sm = smix + H * (kWaKeys + 1);       // [H] maximum
  float* sl = sm + H;                         // [H] sum
  float* st = sl + H;                         // [H, H] mixing matrix
  const int t = blockIdx.x, tid = threadIdx.x;
  const RowMap map{reinterpret_cast<const int4*>(p.rows), p.seq_lens};
  const int4 r = map.get(t);
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo;
  const int pos = r.y;
  if (pos < 0) {
    for (int i = tid; i < H * D; i += kWaThreads) stf(out + i, 0.f);
    return;
  }
  if (pos >= p.qscale_len) {
    if (tid == 0) report_status(p.status, kStatusBadIndex);
    return;
  }
  const float qs = p.qscale[pos];
  const T* q = reinterpret_cast<const T*>(p.q) + (size_t)t * p.ldq;
  for (int i = tid; i < H * D; i += kWaThreads) {
    sq[i] = ldf(q + i);
    sacc[i] = 0.f;
  }
  for (int i = tid; i < H; i += kWaThreads) {
    sm[i] = -INFINITY;
    sl[i] = 0.f;
  }
  if (p.talk != nullptr)
    for (int i = tid; i < H * H; i += kWaThreads) st[i] = ldf(reinterpret_cast<const T*>(p.talk) + i);
  const T* kc = reinterpret_cast<const T*>(p.k_cache);
  const int* table = p.block_tables + (size_t)r.x * p.max_blocks;
  const int lo = pos - p.window + 1 > 0 ? pos - p.window + 1 : 0;

  auto stage = [&](int m, int j0, int n) {
    for (int i = tid; i < n * (D / 8); i += kWaThreads) {
      const int key = i / (D / 8), d = (i % (D / 8)) * 8, j = j0 + key;
      int blk = table[j / p.block_size];
      if (blk < 0 || blk >= p.num_cache_blocks) {
        report_status(p.status, kStatusBadIndex);
        blk = 0;
      }
      float v[8];
      ld8(kc + (((size_t)blk * G + m) * p.block_size + j % p.block_size) * D + d, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) sk[key * kp + d + e] = v[e];
    }
  };
  auto scores = [&](int m, int j0, int n) {  // sw of the heads that read key head m
    for (int i = tid; i < grp * kWaKeys; i += kWaThreads) {
      const int h = m * grp + i / kWaKeys, key = i % kWaKeys;
      float s = -INFINITY;
      if (key < n) {
        const float* a = sq + h * D;
        const float* b = sk + key * kp;
        float acc = 0.f;
        for (int d = 0; d < D; ++d) acc = fmaf(a[d], b[d], acc);
        const int dist = pos - (j0 + key);
        s = acc * qs - p.bias[(size_t)h * p.bias_len + dist];
      }
      sw[h * (kWaKeys + 1) + key] = s;
    }
  };

  for (int j0 = lo; j0 <= pos; j0 += kWaKeys) {
    const int n = pos - j0 + 1 < kWaKeys ? pos - j0 + 1 : kWaKeys;
    for (int m = 0; m < G; ++m) {
      __syncthreads();
      stage(m, j0, n);
      __syncthreads();
      scores(m, j0, n);
    }
    __syncthreads();
    for (int h = tid; h < H; h += kWaThreads) {
      float mx = sm[h];
      for (int key = 0; key < n; ++key) mx = fmaxf(mx, sw[h * (kWaKeys + 1) + key]);
      float l = sl[h] * exp2f(sm[h] - mx);
      for (int key = 0; key < n; ++key) l += exp2f(sw[h * (kWaKeys + 1) + key] - mx);
      sm[h] = mx;
      sl[h] = l;
    }
  }
  for (int j0 = lo; j0 <= pos; j0 += kWaKeys) {
    const int n = pos - j0 + 1 < kWaKeys ? pos - j0 + 1 : kWaKeys;
    for (int m = 0; m < G; ++m) {
      __syncthreads();
      stage(m, j0, n);
      __syncthreads();
      scores(m, j0, n);
    }
    __syncthreads();
    for (int i = tid; i < H * kWaKeys; i += kWaThreads) {
      const int h = i / kWaKeys, key = i % kWaKeys;
      float& w = sw[h * (kWaKeys + 1) + key];
      w = key < n ? exp2f(w - sm[h]) / sl[h] : 0.f;
    }
    __syncthreads();
    const float* wts = sw;
    if (p.talk != nullptr) {
      for (int i = tid; i < H * kWaKeys; i += kWaThreads) {
        const int h = i / kWaKeys, key = i % kWaKeys;
        float acc = 0.f;
        for (int g = 0; g < H; ++g) acc = fmaf(st[h * H + g], sw[g * (kWaKeys + 1) + key], acc);
        smix[h * (kWaKeys + 1) + key] = acc;
      }
      wts = smix;
    }
    for (int m = 0; m < G; ++m) {
      if (G > 1 || m > 0) {  // with one key head its keys are still staged
        __syncthreads();
        stage(m, j0, n);
      }
      __syncthreads();
      for (int i = tid; i < grp * D; i += kWaThreads) {
        const int h = m * grp + i / D, d = i % D;
        float acc = sacc[h * D + d];
        for (int key = 0; key < n; ++key) acc = fmaf(wts[h * (kWaKeys + 1) + key], sk[key * kp + d], acc);
        sacc[h * D + d] = acc;
      }
    }
  }
  __syncthreads();
  const T* gate = p.gate != nullptr ? reinterpret_cast<const T*>(p.gate) + (size_t)t * p.ldg : nullptr;
  for (int i = tid; i < H * D; i += kWaThreads) {
    float v = sacc[i];
    if (gate != nullptr) v *= 1.f / (1.f + expf(-ldf(gate + i)));
    stf(out + i, v);
  }
}

// ------------------------------------------------------------------------------------------------
// fp32 GEMM on the CUDA cores: 64 x 64 tile, 4 x 4 outputs per thread, K in order.
constexpr int kFT = 64, kFK = 16;

struct F32Store {
  float* d;
  long long ldd;
  GemmF32Post post;
  __device__ __forceinline__ void operator()(int row, int col, float v, float) const {
    float& o = d[(size_t)row * ldd + col];
    if (post.relu2) v = v > 0.f ? v * v : 0.f;
    if (post.softcap > 0.f) v = post.softcap * tanhf(v / post.softcap);
    o = post.accumulate ? o + v : v;
  }
};
struct F32Swiglu {
  float* d;
  long long ldd;
  __device__ __forceinline__ void operator()(int row, int col, float g, float u) const {
    d[(size_t)row * ldd + col] = g / (1.f + expf(-g)) * u;
  }
};
struct F32Dyt {
  float* x;
  long long ldx;
  float* h;
  long long ldh;
  DytNorm<float> n1, n2;
  __device__ __forceinline__ void operator()(int row, int col, float v, float) const {
    float& xr = x[(size_t)row * ldx + col];
    const float nx = xr + fmaf(tanhf(*n1.alpha * v), n1.w[col], n1.b[col]);
    xr = nx;
    h[(size_t)row * ldh + col] = fmaf(tanhf(*n2.alpha * nx), n2.w[col], n2.b[col]);
  }
};

template <bool DUAL, class Epi>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ a, long long lda, const float* __restrict__ b,
                                                       long long ldb, int M, int N, int K, Epi epi) {
  __shared__ float sa[kFK][kFT + 4], sb[kFK][kFT + 4], sb2[DUAL ? kFK : 1][kFT + 4];
  const int m0 = blockIdx.y * kFT, n0 = blockIdx.x * kFT;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4], acc2[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = acc2[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += kFK) {
    for (int i = threadIdx.x; i < kFT * kFK; i += 256) {
      const int r = i / kFK, k = i % kFK;
      const bool kin = k0 + k < K;
      sa[k][r] = (kin && m0 + r < M) ? a[(size_t)(m0 + r) * lda + k0 + k] : 0.f;
      sb[k][r] = (kin && n0 + r < N) ? b[(size_t)(n0 + r) * ldb + k0 + k] : 0.f;
      if constexpr (DUAL) sb2[k][r] = (kin && n0 + r < N) ? b[(size_t)(N + n0 + r) * ldb + k0 + k] : 0.f;
    }
    __syncthreads();
    // sums of kFK products first, then the sum of those: the rounding error of a long K stays that of a short one
    float part[4][4], part2[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) part[i][j] = part2[i][j] = 0.f;
#pragma unroll
    for (int k = 0; k < kFK; ++k) {
      float av[4], bv[4], cv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        av[i] = sa[k][ty * 4 + i];
        bv[i] = sb[k][tx * 4 + i];
        if constexpr (DUAL) cv[i] = sb2[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          part[i][j] = fmaf(av[i], bv[j], part[i][j]);
          if constexpr (DUAL) part2[i][j] = fmaf(av[i], cv[j], part2[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[i][j] += part[i][j];
        if constexpr (DUAL) acc2[i][j] += part2[i][j];
      }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int row = m0 + ty * 4 + i;
    if (row >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = n0 + tx * 4 + j;
      if (col < N) epi(row, col, acc[i][j], acc2[i][j]);
    }
  }
}

template <bool DUAL, class Epi>
void run_gemm_f32(const float* a, long long lda, const float* b, long long ldb, int M, int N, int K, const Epi& e, cudaStream_t s) {
  if (M == 0 || N == 0) return;
  dim3 grid((N + kFT - 1) / kFT, (M + kFT - 1) / kFT);
  gemm_f32_kernel<DUAL, Epi><<<grid, 256, 0, s>>>(a, lda, b, ldb, M, N, K, e);
  check_cuda(cudaGetLastError(), "gemm_f32");
}

// ------------------------------------------------------------------------------------------------
__device__ __forceinline__ uint32_t mix_u32(uint32_t x) {  // the noise hash of the fused lm_head sampler
  x ^= x >> 16;
  x *= 0x7feb352dU;
  x ^= x >> 15;
  x *= 0x846ca68bU;
  x ^= x >> 16;
  return x;
}
__global__ void __launch_bounds__(256) sample_logits_kernel(const float* __restrict__ logits, long long ld, int V, float inv_temp, int greedy,
                                                            const unsigned long long* __restrict__ seeds, int* __restrict__ tokens,
                                                            float* __restrict__ logprobs) {
  __shared__ float s_best[256], s_z[256], s_m[256], s_s[256];
  __shared__ int s_idx[256];
  const int row = blockIdx.x, tid = threadIdx.x;
  const unsigned long long sd = seeds[row];
  const uint32_t lo = (uint32_t)sd, hi = (uint32_t)(sd >> 32);
  float best = -INFINITY, bz = 0.f, m = -INFINITY, sum = 0.f;
  int idx = 0x7fffffff;
  for (int c = tid; c < V; c += 256) {
    const float z = logits[(size_t)row * ld + c] * inv_temp;
    float v = z;
    if (!greedy) {
      const float u = ((float)(mix_u32(mix_u32((uint32_t)c ^ lo) + hi) >> 8) + 0.5f) * (1.0f / 16777216.0f);
      v += -logf(-logf(u));
    }
    if (v > best) {
      best = v;
      bz = z;
      idx = c;
    }
    if (z > m) {
      sum = sum * expf(m - z) + 1.f;
      m = z;
    } else {
      sum += expf(z - m);
    }
  }
  s_best[tid] = best; s_z[tid] = bz; s_m[tid] = m; s_s[tid] = sum; s_idx[tid] = idx;
  __syncthreads();
  for (int o = 128; o > 0; o >>= 1) {
    if (tid < o) {
      const int j = tid + o;
      if (s_best[j] > s_best[tid] || (s_best[j] == s_best[tid] && s_idx[j] < s_idx[tid])) {
        s_best[tid] = s_best[j];
        s_z[tid] = s_z[j];
        s_idx[tid] = s_idx[j];
      }
      const float nm = fmaxf(s_m[tid], s_m[j]);
      const float a = s_m[tid] == -INFINITY ? 0.f : s_s[tid] * expf(s_m[tid] - nm);
      const float b = s_m[j] == -INFINITY ? 0.f : s_s[j] * expf(s_m[j] - nm);
      s_s[tid] = a + b;
      s_m[tid] = nm;
    }
    __syncthreads();
  }
  if (tid == 0) {
    tokens[row] = s_idx[0] == 0x7fffffff ? 0 : s_idx[0];
    if (logprobs != nullptr) logprobs[row] = s_z[0] - (s_m[0] + logf(s_s[0]));
  }
}

template <typename T>
void window_attn_t(const WindowAttnArgs& a, cudaStream_t s) {
  const size_t smem = sizeof(float) * ((size_t)2 * a.H * a.D + kWaKeys * (a.D + 1) + 2 * a.H * (kWaKeys + 1) + 2 * a.H + (size_t)a.H * a.H);
  if (smem > 220 * 1024) throw std::runtime_error("window_attn: heads x head size too large");
  auto kernel = window_attn_kernel<T>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, 220 * 1024, "window_attn smem attr");
  launch_kernel(kernel, dim3(a.T), dim3(kWaThreads), smem, s, "window_attn", a);
}

}  // namespace

void launch_embed_dyt(bool fp32, const int* ids, const void* table, float scale, float* x, void* h, const DytArgs& norm, int T, int W, int V,
                      cudaStream_t s) {
  if (T == 0) return;
  const dim3 grid((T + 3) / 4), block(128);
  if (fp32) {
    AGRPO_PREFER_SMEM(embed_dyt_kernel<float>);
    launch_kernel(embed_dyt_kernel<float>, grid, block, 0, s, "embed_dyt", ids, (const float*)table, scale, x, (float*)h, as_norm<float>(norm), T, W, V);
  } else {
    AGRPO_PREFER_SMEM(embed_dyt_kernel<bf16>);
    launch_kernel(embed_dyt_kernel<bf16>, grid, block, 0, s, "embed_dyt", ids, (const bf16*)table, scale, x, (bf16*)h, as_norm<bf16>(norm), T, W, V);
  }
}

namespace {
template <typename T>
void short_conv_t(const ShortConvArgs& a, cudaStream_t s) {
  const dim3 grid((a.T + kConvRows - 1) / kConvRows, ((a.q_cols + a.k_cols) / 8 + 127) / 128), block(128);
  auto kernel = a.taps == 1 ? short_conv_kernel<T, 1> : a.taps == 2 ? short_conv_kernel<T, 2> : a.taps == 3 ? short_conv_kernel<T, 3>
                : a.taps == 4 ? short_conv_kernel<T, 4> : short_conv_kernel<T, 0>;
  launch_kernel(kernel, grid, block, 0, s, "short_conv", a);
}
}  // namespace

void launch_short_conv_decode(bool fp32, const ShortConvArgs& a, cudaStream_t s) {
  if (a.T == 0) return;
  if (a.ring_len < a.taps) throw std::runtime_error("short_conv: ring shorter than the taps");
  const dim3 grid(a.T, ((a.q_cols + a.k_cols) / 8 + 127) / 128), block(128);
  launch_kernel(fp32 ? short_conv_decode_kernel<float> : short_conv_decode_kernel<bf16>, grid, block, 0, s, "short_conv_decode", a);
}

void launch_short_conv(bool fp32, const ShortConvArgs& a, cudaStream_t s) {
  if (a.T == 0) return;
  if (fp32) short_conv_t<float>(a, s);
  else short_conv_t<bf16>(a, s);
}

void launch_short_conv_ring(bool fp32, const ShortConvArgs& a, const int* ring_rows, int n_ring_rows, cudaStream_t s) {
  const int n = ring_rows != nullptr ? n_ring_rows : a.T;
  if (n == 0 || a.taps <= 1) return;
  const dim3 grid(n, ((a.q_cols + a.k_cols) / 8 + 127) / 128), block(128);
  if (fp32) launch_kernel(short_conv_ring_kernel<float>, grid, block, 0, s, "short_conv_ring", a, ring_rows);
  else launch_kernel(short_conv_ring_kernel<bf16>, grid, block, 0, s, "short_conv_ring", a, ring_rows);
}

void launch_window_attn(bool fp32, const WindowAttnArgs& a, cudaStream_t s) {
  if (a.T == 0) return;
  if (fp32) window_attn_t<float>(a, s);
  else window_attn_t<bf16>(a, s);
}

void launch_gemm_f32(const float* a, long long lda, const float* b, long long ldb, float* d, long long ldd, int M, int N, int K,
                     cudaStream_t s, const GemmF32Post& post) {
  run_gemm_f32<false>(a, lda, b, ldb, M, N, K, F32Store{d, ldd, post}, s);
}
void launch_gemm_swiglu_f32(const float* a, long long lda, const float* b, long long ldb, float* d, long long ldd, int M, int F, int K,
                            cudaStream_t s) {
  run_gemm_f32<true>(a, lda, b, ldb, M, F, K, F32Swiglu{d, ldd}, s);
}
void launch_gemm_dyt_f32(const float* a, long long lda, const float* b, long long ldb, int M, int N, int K, float* x, long long ldx,
                         float* h, long long ldh, const DytArgs& n1, const DytArgs& n2, cudaStream_t s) {
  run_gemm_f32<false>(a, lda, b, ldb, M, N, K, F32Dyt{x, ldx, h, ldh, as_norm<float>(n1), as_norm<float>(n2)}, s);
}

void launch_sample_logits(const float* logits, long long ld, int rows, int V, float temperature, const unsigned long long* seeds,
                          int* tokens, float* logprobs, cudaStream_t s) {
  if (rows == 0) return;
  const int greedy = temperature <= 0.f ? 1 : 0;
  sample_logits_kernel<<<rows, 256, 0, s>>>(logits, ld, V, greedy ? 1.f : 1.f / temperature, greedy, seeds, tokens, logprobs);
  check_cuda(cudaGetLastError(), "sample_logits");
}

}  // namespace agrpo
