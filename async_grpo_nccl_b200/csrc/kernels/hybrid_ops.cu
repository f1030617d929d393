// Operations of hybrid attention / scan decoders in their plain form, for bf16 and for 32-bit activations: embedding with the
// following norms, zero-centred RMS norms, norm + rotation + cache write of whole query / key projections, attention inside
// position chunks (any head size), and the selective scan (any sizes). Built without fast-math.
#include "../common/ptx.cuh"
#include "../launchers.h"
#include "../launchers_hybrid.h"
#include "layer_ops.cuh"

namespace agrpo {

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Eight channels of one consumer: x * scale * (1 + w).
template <typename T>
__device__ __forceinline__ void norm_out8(const NormOut& o, size_t row, int c, const float (&x)[8], float scale) {
  if (o.h == nullptr) return;
  float w[8], y[8];
  if (o.w != nullptr) {
    ld8(reinterpret_cast<const T*>(o.w) + c, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = x[i] * scale * (1.f + w[i]);
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = x[i];
  }
  st8(reinterpret_cast<T*>(o.h) + row * o.ld + c, y);
}

template <typename T>
__global__ void __launch_bounds__(128) embed_norm_kernel(EmbedArgs p) {
  pdl_wait();
  pdl_launch();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= p.T) return;
  int id = p.ids[row];
  id = id < 0 ? 0 : (id >= p.V ? p.V - 1 : id);
  float sq = 0.f;
  for (int c = lane * 8; c < p.W; c += 256) {
    float e[8];
    ld8(reinterpret_cast<const T*>(p.table) + (size_t)id * p.W + c, e);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      e[i] *= p.scale;
      sq += e[i] * e[i];
    }
    st8(p.x + (size_t)row * p.W + c, e);
    if (p.copy != nullptr) st8(reinterpret_cast<T*>(p.copy) + (size_t)row * p.ld_copy + c, e);
    norm_out8<T>(p.out[0], row, c, e, 1.f);
    norm_out8<T>(p.out[1], row, c, e, 1.f);
  }
  sq = warp_sum(sq);
  if (p.ss != nullptr)
    for (int i = lane; i < p.n_stats; i += 32) p.ss[(size_t)i * p.ss_pitch + row] = i == 0 && p.out[0].w != nullptr ? sumsq_to_fixed(sq) : 0;
}

template <typename T>
__global__ void __launch_bounds__(128) rms_rows_kernel(const float* __restrict__ x, long long ldx, NormOut o0, NormOut o1, float eps, int width,
                                                       int T_, int W) {
  pdl_wait();
  pdl_launch();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= T_) return;
  const float* src = x + (size_t)row * ldx;
  float sq = 0.f;
  for (int c = lane * 8; c < W; c += 256) {
    float v[8];
    ld8(src + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) sq += v[i] * v[i];
  }
  const float scale = 1.f / sqrtf(warp_sum(sq) / (float)width + eps);
  for (int c = lane * 8; c < W; c += 256) {
    float v[8];
    ld8(src + c, v);
    norm_out8<T>(o0, row, c, v, scale);
    norm_out8<T>(o1, row, c, v, scale);
  }
}

__global__ void softcap_rows_kernel(float* z, long long ld, int V, float cap) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= V) return;
  float& v = z[(size_t)blockIdx.y * ld + c];
  v = cap * tanhf(v / cap);
}

// ------------------------------------------------------------------------------------------------
// CTA = token row. Work item = two runs of eight paired dimensions of a head (or one run of the part that is not rotated); runs that
// do not fit the pairing (odd halves) go one dimension at a time.
constexpr int kQkThreads = 128;

template <typename T>
__global__ void __launch_bounds__(kQkThreads) qk_norm_rope_kernel(QkRopeArgs p) {
  pdl_wait();
  pdl_launch();
  __shared__ float s_part[2][kQkThreads / 32];
  const int t = blockIdx.x, tid = threadIdx.x;
  const RowMap map{reinterpret_cast<const int4*>(p.rows), p.seq_lens};
  const int4 r = map.get(t);
  const int pos = r.y;
  if (pos < 0) return;
  if (pos >= p.max_pos) {
    if (tid == 0) report_status(p.status, kStatusBadIndex);
    return;
  }
  const int blk = p.block_tables[(size_t)r.x * p.max_blocks + pos / p.block_size];
  if (blk < 0 || blk >= p.num_cache_blocks) {
    if (tid == 0) report_status(p.status, kStatusBadIndex);
    return;
  }
  T* u = reinterpret_cast<T*>(p.u) + (size_t)t * p.ldu;
  const int D = p.D, qd = p.H * D, kd = p.G * D;
  float sq = 0.f, sk = 0.f;
  if (p.ss_q != nullptr) {
    sq = sumsq_from_fixed(p.ss_q[t]);
    sk = sumsq_from_fixed(p.ss_k[t]);
  } else {
    for (int c = tid * 8; c < qd + kd; c += kQkThreads * 8) {
      float v[8], s = 0.f;
      ld8(u + c, v);
#pragma unroll
      for (int i = 0; i < 8; ++i) s += v[i] * v[i];
      if (c < qd) sq += s;
      else sk += s;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((tid & 31) == 0) {
      s_part[0][tid >> 5] = sq;
      s_part[1][tid >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
    for (int w = 0; w < kQkThreads / 32; ++w) {
      sq += s_part[0][w];
      sk += s_part[1][w];
    }
  }
  const float iq = 1.f / sqrtf(sq / (float)(p.H * p.dim) + p.eps), ik = 1.f / sqrtf(sk / (float)(p.G * p.dim) + p.eps);
  const int half = p.rot / 2;
  const float* ct = p.cos_t + (size_t)pos * half;
  const float* st = p.sin_t + (size_t)pos * half;
  const T* qn = reinterpret_cast<const T*>(p.q_norm);
  const T* kn = reinterpret_cast<const T*>(p.k_norm);
  T* kc = reinterpret_cast<T*>(p.k_cache) + ((size_t)blk * p.G * p.block_size + pos % p.block_size) * D;
  const size_t head_pitch = (size_t)p.block_size * D;
  if (half % 8 == 0) {
    const int runs = half / 8, rest = (D - 2 * half) / 8, per = runs + rest;
    for (int i = tid; i < (p.H + p.G) * per; i += kQkThreads) {
      const int h = i / per, j = i % per;
      const bool is_q = h < p.H;
      const float inv = is_q ? iq : ik;
      T* src = u + (size_t)h * D;
      const T* w = is_q ? qn + (size_t)h * D : kn + (size_t)(h - p.H) * D;
      T* dst = is_q ? src : kc + (size_t)(h - p.H) * head_pitch;
      if (j < runs) {
        const int d = j * 8;
        float a[8], b[8], wa[8], wb[8], x[8], y[8], c[8], s[8];
        ld8(src + d, a);
        ld8(src + half + d, b);
        ld8(w + d, wa);
        ld8(w + half + d, wb);
        ld8(ct + d, c);
        ld8(st + d, s);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float ua = a[e] * inv * wa[e], ub = b[e] * inv * wb[e];
          x[e] = ua * c[e] - ub * s[e];
          y[e] = ub * c[e] + ua * s[e];
        }
        st8(dst + d, x);
        st8(dst + half + d, y);
      } else {
        const int d = 2 * half + (j - runs) * 8;
        float a[8], wa[8];
        ld8(src + d, a);
        ld8(w + d, wa);
#pragma unroll
        for (int e = 0; e < 8; ++e) a[e] *= inv * wa[e];
        st8(dst + d, a);
      }
    }
  } else {
    const int per = half + (D - 2 * half);
    for (int i = tid; i < (p.H + p.G) * per; i += kQkThreads) {
      const int h = i / per, j = i % per;
      const bool is_q = h < p.H;
      const float inv = is_q ? iq : ik;
      T* src = u + (size_t)h * D;
      const T* w = is_q ? qn + (size_t)h * D : kn + (size_t)(h - p.H) * D;
      T* dst = is_q ? src : kc + (size_t)(h - p.H) * head_pitch;
      if (j < half) {
        const float ua = ldf(src + j) * inv * ldf(w + j), ub = ldf(src + half + j) * inv * ldf(w + half + j);
        stf(dst + j, ua * ct[j] - ub * st[j]);
        stf(dst + half + j, ub * ct[j] + ua * st[j]);
      } else {
        const int d = half + j;
        stf(dst + d, ldf(src + d) * inv * ldf(w + d));
      }
    }
  }
  T* vc = reinterpret_cast<T*>(p.v_cache) + ((size_t)blk * p.G * p.block_size + pos % p.block_size) * p.E;
  for (int i = tid; i < p.G * p.E / 8; i += kQkThreads) {
    const int g = i / (p.E / 8), d = (i % (p.E / 8)) * 8;
    float v[8];
    ld8(u + qd + kd + g * p.E + d, v);
    st8(vc + (size_t)g * p.block_size * p.E + d, v);
  }
}

// ------------------------------------------------------------------------------------------------
// Attention inside a chunk, CTA = (head, token row): the four warps take every fourth key, lanes share the dimensions, and the
// warps' running (maximum, sum, output) are merged at the end.
constexpr int kCaDims = 16;  // dimensions per lane: heads up to 512

template <typename T>
__global__ void __launch_bounds__(128) chunk_attn_kernel(ChunkAttnArgs p) {
  pdl_wait();
  pdl_launch();
  extern __shared__ float ca_smem[];  // [4][E] outputs, [4] maxima, [4] sums
  const int h = blockIdx.x, t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = h / (p.H / p.G), D = p.D, E = p.E;
  const RowMap map{reinterpret_cast<const int4*>(p.rows), p.seq_lens};
  const int4 r = map.get(t);
  const int pos = r.y;
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo + (size_t)h * E;
  if (pos < 0) {
    for (int i = threadIdx.x; i < E; i += 128) stf(out + i, 0.f);
    return;
  }
  const T* q = reinterpret_cast<const T*>(p.q) + (size_t)t * p.ldq + (size_t)h * D;
  const int* table = p.block_tables + (size_t)r.x * p.max_blocks;
  float qv[kCaDims], acc[kCaDims];
#pragma unroll
  for (int i = 0; i < kCaDims; ++i) {
    qv[i] = i * 32 + lane < D ? ldf(q + i * 32 + lane) : 0.f;
    acc[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const int lo = pos / p.chunk * p.chunk;
  for (int j = lo + warp; j <= pos; j += 4) {
    int blk = table[j / p.block_size];
    if (blk < 0 || blk >= p.num_cache_blocks) {
      report_status(p.status, kStatusBadIndex);
      blk = 0;
    }
    const size_t slot = ((size_t)blk * p.G + g) * p.block_size + j % p.block_size;
    const T* k = reinterpret_cast<const T*>(p.k_cache) + slot * D;
    const T* v = reinterpret_cast<const T*>(p.v_cache) + slot * E;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < kCaDims; ++i)
      if (i * 32 + lane < D) s = fmaf(qv[i], ldf(k + i * 32 + lane), s);
    s = warp_sum(s) * p.scale;
    if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
    const float m_new = fmaxf(m, s);
    const float keep = expf(m - m_new), w = expf(s - m_new);
    l = l * keep + w;
    m = m_new;
#pragma unroll
    for (int i = 0; i < kCaDims; ++i)
      if (i * 32 + lane < E) acc[i] = fmaf(w, ldf(v + i * 32 + lane), acc[i] * keep);
  }
  float* so = ca_smem;
  float* sm = so + 4 * E;
  float* sl = sm + 4;
#pragma unroll
  for (int i = 0; i < kCaDims; ++i)
    if (i * 32 + lane < E) so[warp * E + i * 32 + lane] = acc[i];
  if (lane == 0) {
    sm[warp] = m;
    sl[warp] = l;
  }
  __syncthreads();
  const float mx = fmaxf(fmaxf(sm[0], sm[1]), fmaxf(sm[2], sm[3]));
  float w[4], total = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    w[i] = sm[i] == -INFINITY ? 0.f : expf(sm[i] - mx);
    total += w[i] * sl[i];
  }
  for (int i = threadIdx.x; i < E; i += 128)
    stf(out + i, (w[0] * so[i] + w[1] * so[E + i] + w[2] * so[2 * E + i] + w[3] * so[3 * E + i]) / total);
}

// ------------------------------------------------------------------------------------------------
// Selective scan, thread = channel of a segment, states in shared memory, token after token.
constexpr int kPlainChannels = 64;

// exp(z) for z <= 0. A state that fades slowly multiplies by numbers just below one many times over, so what counts there is the
// rounding of the last bit: near zero the Taylor series, whose last step (one plus a small number) is rounded once.
__device__ __forceinline__ float decay(float z) {
  if (z < -0.5f) return expf(z);
  float p = 1.f / 362880.f;
  p = fmaf(p, z, 1.f / 40320.f);
  p = fmaf(p, z, 1.f / 5040.f);
  p = fmaf(p, z, 1.f / 720.f);
  p = fmaf(p, z, 1.f / 120.f);
  p = fmaf(p, z, 1.f / 24.f);
  p = fmaf(p, z, 1.f / 6.f);
  p = fmaf(p, z, 0.5f);
  p = fmaf(p, z, 1.f);
  return fmaf(p, z, 1.f);
}

template <typename T>
__global__ void __launch_bounds__(kPlainChannels) selective_scan_plain_kernel(ScanArgs p) {
  pdl_wait();
  pdl_launch();
  extern __shared__ float ps_smem[];  // [channels][N + 1]
  const int c = blockIdx.x * kPlainChannels + threadIdx.x;
  if (c >= p.C) return;
  int row0 = blockIdx.y, n = 1, slot = blockIdx.y, pos = 0;
  if (p.segs != nullptr) {
    const int4 s = reinterpret_cast<const int4*>(p.segs)[blockIdx.y];
    row0 = s.x;
    n = s.y;
    slot = s.z;
    pos = s.w;
  } else {
    pos = p.seq_lens[row0] - 1;
    if (pos < 0) return;
  }
  const int N = p.N;
  float* S = ps_smem + threadIdx.x * (N + 1);
  float* st = p.state + (size_t)slot * p.state_pitch + (size_t)c * N;
  for (int i = 0; i < N; ++i) S[i] = pos > 0 ? st[i] : 0.f;
  const T* w = reinterpret_cast<const T*>(p.wdt) + (size_t)c * p.ldw;
  const float* A = p.a + (size_t)c * N;
  for (int t = row0; t < row0 + n; ++t) {
    const float* r = p.r + (size_t)t * p.ldr;
    float v = p.dt_b[c];
    float acc = 0.f;
    for (int i = 0; i < p.rank; ++i) acc = fmaf(ldf(w + i), r[i], acc);
    v += acc;
    const float dt = fmaxf(v, 0.f) + log1pf(expf(-fabsf(v)));
    const float x = ldf(reinterpret_cast<const T*>(p.xc) + (size_t)t * p.ldx + c);
    const float in = dt * x;
    float y = 0.f;
    for (int i = 0; i < N; ++i) {
      const float s = fmaf(decay(dt * A[i]), S[i], in * r[p.rank + i]);
      S[i] = s;
      y = fmaf(s, r[p.rank + N + i], y);
    }
    y = fmaf(p.d[c], x, y);
    const float z = ldf(reinterpret_cast<const T*>(p.z) + (size_t)t * p.ldz + c);
    stf(reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo + c, y * (z / (1.f + expf(-z))));
  }
  for (int i = 0; i < N; ++i) st[i] = S[i];
}

}  // namespace

void launch_embed_norm(bool fp32, const EmbedArgs& a, cudaStream_t s) {
  if (a.T == 0) return;
  const dim3 grid((a.T + 3) / 4), block(128);
  auto kernel = fp32 ? embed_norm_kernel<float> : embed_norm_kernel<bf16>;
  prefer_max_shared(kernel);
  launch_kernel(kernel, grid, block, 0, s, "embed_norm", a);
}

void launch_rms_rows(bool fp32, const float* x, long long ldx, const NormOut out[2], float eps, int width, int T, int W, cudaStream_t s) {
  if (T == 0) return;
  const dim3 grid((T + 3) / 4), block(128);
  auto kernel = fp32 ? rms_rows_kernel<float> : rms_rows_kernel<bf16>;
  prefer_max_shared(kernel);
  launch_kernel(kernel, grid, block, 0, s, "rms_rows", x, ldx, out[0], out[1], eps, width, T, W);
}

void launch_softcap_rows(float* z, long long ld, int rows, int V, float cap, cudaStream_t s) {
  if (rows == 0 || cap <= 0.f) return;
  softcap_rows_kernel<<<dim3((V + 255) / 256, rows), 256, 0, s>>>(z, ld, V, cap);
  check_cuda(cudaGetLastError(), "softcap_rows");
}

void launch_qk_norm_rope(bool fp32, const QkRopeArgs& a, cudaStream_t s) {
  if (a.T == 0) return;
  auto kernel = fp32 ? qk_norm_rope_kernel<float> : qk_norm_rope_kernel<bf16>;
  prefer_max_shared(kernel);
  launch_kernel(kernel, dim3(a.T), dim3(kQkThreads), 0, s, "qk_norm_rope", a);
}

void launch_chunk_attn(bool fp32, const ChunkAttnArgs& a, cudaStream_t s) {
  if (a.T == 0) return;
  if (a.D > 32 * kCaDims || a.E > 32 * kCaDims) throw std::runtime_error("chunk_attn: heads up to 512");
  const size_t smem = (4 * (size_t)a.E + 8) * sizeof(float);
  for (int t0 = 0; t0 < a.T; t0 += 32768) {  // grid.y limit; a row table shifts with the rows
    if (t0 > 0 && a.rows == nullptr) throw std::runtime_error("chunk_attn: too many decode rows");
    ChunkAttnArgs p = a;
    const size_t es = fp32 ? 4 : 2;
    p.T = a.T - t0 < 32768 ? a.T - t0 : 32768;
    p.q = reinterpret_cast<const char*>(a.q) + (size_t)t0 * a.ldq * es;
    p.out = reinterpret_cast<char*>(a.out) + (size_t)t0 * a.ldo * es;
    if (a.rows != nullptr) p.rows = a.rows + (size_t)t0 * 4;
    launch_kernel(fp32 ? chunk_attn_kernel<float> : chunk_attn_kernel<bf16>, dim3(p.H, p.T), dim3(128), smem, s, "chunk_attn", p);
  }
}

void launch_selective_scan_plain(bool fp32, const ScanArgs& a, cudaStream_t s) {
  const int n = a.segs != nullptr ? a.n_segs : a.T;
  if (n == 0) return;
  const size_t smem = (size_t)kPlainChannels * (a.N + 1) * sizeof(float);
  if (smem > 220 * 1024) throw std::runtime_error("selective_scan: too many states per channel");
  auto kernel = fp32 ? selective_scan_plain_kernel<float> : selective_scan_plain_kernel<bf16>;
  check_cuda(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024), "selective_scan_plain smem attr");
  launch_kernel(kernel, dim3((a.C + kPlainChannels - 1) / kPlainChannels, n), dim3(kPlainChannels), smem, s, "selective_scan_plain", a);
}

}  // namespace agrpo
