// Attention inside position chunks with soft-capped scores on the tensor cores, over paged keys and values.
//
// A capped score lies in [-cap, cap]. Where cap is small enough for exp(cap) and exp(-cap) to stay far inside the range of fp32
// (and of bf16, which has the same exponents), the softmax needs no maximum: weights are exp(score), sums and products are
// accumulated as they come, and the division by the sum at the end cancels the scale. Scores are then read once and nothing is
// ever rescaled. Larger caps, or none, take the running maximum.
#include <cuda_bf16.h>
#include <math.h>

#include "../common/ptx.cuh"
#include "../common/tensormap.h"
#include "../launchers.h"
#include "../launchers_hybrid.h"
#include "decode_attn.cuh"
#include "layer_ops.cuh"

namespace agrpo {

namespace {

typedef __nv_bfloat16 bf16;
typedef unsigned long long f32x2;

constexpr float kLog2e = 1.4426950408889634f;
constexpr float kFreeCap = 66.f;   // exp(+-66) is 2^(+-95): room for sums over 2^20 keys of values up to 2^10

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
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Score in log2 units of a raw product. t = product * in; capped: out * tanh(t), else t itself (in = scale * log2 e).
struct CapScale {
  float in, out;   // out 0: no cap
  __device__ __forceinline__ float operator()(float raw) const {
    const float t = raw * in;
    return out > 0.f ? out * tanh_f32(t) : t;
  }
};
inline CapScale cap_scale(float scale, float cap) {
  CapScale c;
  c.in = cap > 0.f ? scale / cap : scale * kLog2e;
  c.out = cap > 0.f ? cap * kLog2e : 0.f;
  return c;
}

// ================================================================================================
// Prompts: CTA = 128 query rows of one head. S and O live in tensor memory, keys and values arrive by TMA from matrices that the
// step's pages were gathered into, P goes back over S as bf16 and is the A operand of P V. Two CTAs fit an SM, so that one's
// softmax overlaps the other's products.
// ================================================================================================
constexpr int kBM = 128;
constexpr int kBN = 128;
constexpr int kThreads = 192;

struct ChunkPrefillParams {
  const int4* tiles;   // {first row, rows, position of the first row, row of position 0 among the gathered keys}
  bf16* out;
  long long ldo;
  int group, chunk;
  CapScale sc;
  int* status;
};

// 32 raw scores -> weights (not normalised); adds them to l. Small arguments of tanh (the usual case) take the odd series up to
// z^9, two at a time; if any score of the warp is larger, all take the exponential form.
template <bool MASKED>
__device__ __forceinline__ void free_weights(const uint32_t (&s)[32], const CapScale& sc, int lo, int hi, uint32_t (&w)[16], float& l) {
  float mx[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 32; ++i) mx[i & 3] = fmaxf(mx[i & 3], fabsf(__uint_as_float(s[i])));
  const bool small = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * fabsf(sc.in) <= 0.25f;
  float l0 = 0.f, l1 = 0.f;
  if (__all_sync(0xffffffffu, small)) {
    const f32x2 in = pack2(sc.in, sc.in);
    const f32x2 c0 = pack2(sc.out, sc.out), c1 = pack2(sc.out * (-1.f / 3.f), sc.out * (-1.f / 3.f)), c2 = pack2(sc.out * (2.f / 15.f), sc.out * (2.f / 15.f)),
                c3 = pack2(sc.out * (-17.f / 315.f), sc.out * (-17.f / 315.f)), c4 = pack2(sc.out * (62.f / 2835.f), sc.out * (62.f / 2835.f));
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      const f32x2 t = mul2(pack2(__uint_as_float(s[2 * i]), __uint_as_float(s[2 * i + 1])), in);
      const f32x2 y = mul2(t, t);
      const f32x2 e = mul2(t, fma2(fma2(fma2(fma2(c4, y, c3), y, c2), y, c1), y, c0));
      float a, b;
      unpack2(e, a, b);
      a = ex2(a);
      b = ex2(b);
      if (MASKED) {
        if (2 * i < lo || 2 * i > hi) a = 0.f;
        if (2 * i + 1 < lo || 2 * i + 1 > hi) b = 0.f;
      }
      l0 += a;
      l1 += b;
      w[i] = pack_bf16x2(a, b);
    }
  } else {
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float a = ex2(sc.out * tanh_abs_f32(__uint_as_float(s[2 * i]) * sc.in));
      float b = ex2(sc.out * tanh_abs_f32(__uint_as_float(s[2 * i + 1]) * sc.in));
      if (MASKED) {
        if (2 * i < lo || 2 * i > hi) a = 0.f;
        if (2 * i + 1 < lo || 2 * i + 1 > hi) b = 0.f;
      }
      l0 += a;
      l1 += b;
      w[i] = pack_bf16x2(a, b);
    }
  }
  l += l0 + l1;
}

template <int D, int E, bool FREE>
__global__ void __launch_bounds__(kThreads, 2)
chunk_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                     const ChunkPrefillParams p) {
  constexpr int kQBytes = kBM * D * 2, kKBytes = kBN * D * 2, kVBytes = kBN * E * 2;
  constexpr uint32_t kTmemCols = 256;
  constexpr uint32_t kIdescS = umma_idesc_bf16(kBM, kBN, 0, 0);
  constexpr uint32_t kIdescO = umma_idesc_bf16(kBM, E, 0, 1);
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + kQBytes;
  uint8_t* sV = sK + kKBytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + kVBytes);
  uint64_t* q_full = bars + 0;
  uint64_t* k_full = bars + 1;
  uint64_t* v_full = bars + 2;
  uint64_t* s_full = bars + 3;
  uint64_t* p_ready = bars + 4;
  uint64_t* o_done = bars + 5;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 6);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.x, kv_head = head / p.group;
  const int4 tile = p.tiles[blockIdx.y];
  const int pos0 = tile.z, n_rows = tile.y;
  const int j0 = pos0 / p.chunk * p.chunk;                 // oldest key that the first row sees
  const int n_kv = (pos0 + n_rows - j0 + kBN - 1) / kBN;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(k_full, 1);
    mbar_init(v_full, 1);
    mbar_init(s_full, 1);
    mbar_init(p_ready, 4);
    mbar_init(o_done, 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_wait();
  pdl_launch();
  const uint32_t tmem_S = *tmem_slot;
  const uint32_t tmem_O = tmem_S + 128;

  if (warp == 0) {
    if (elect_one()) {
      mbar_expect_tx(q_full, kQBytes);
#pragma unroll
      for (int c = 0; c < D / 64; ++c) tma_load_2d(sQ + c * (kBM * 128), &tmQ, q_full, head * D + c * 64, tile.x);
      for (int j = 0; j < n_kv; ++j) {
        const int row = tile.w + j0 + j * kBN;  // rows past the gathered keys read as zero, other segments' rows are masked
        if (j > 0 && !mbar_wait(s_full, (j - 1) & 1)) {
          report_status(p.status, kStatusWaitEmptyTimeout);
          break;
        }
        mbar_expect_tx(k_full, kKBytes);
#pragma unroll
        for (int c = 0; c < D / 64; ++c) tma_load_2d(sK + c * (kBN * 128), &tmK, k_full, kv_head * D + c * 64, row);
        if (j > 0 && !mbar_wait(o_done, (j - 1) & 1)) {
          report_status(p.status, kStatusWaitEmptyTimeout);
          break;
        }
        mbar_expect_tx(v_full, kVBytes);
#pragma unroll
        for (int c = 0; c < E / 64; ++c) tma_load_2d(sV + c * (kBN * 128), &tmV, v_full, kv_head * E + c * 64, row);
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      bool ok = mbar_wait(q_full, 0);
      if (!ok) report_status(p.status, kStatusWaitFullTimeout);
      const uint32_t aQ = smem_u32(sQ), aK = smem_u32(sK), aV = smem_u32(sV);
      for (int j = 0; j < n_kv && ok; ++j) {
        if (!mbar_wait(k_full, j & 1)) {
          report_status(p.status, kStatusWaitFullTimeout);
          break;
        }
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < D / 16; ++k) {
          const uint32_t off = (k / 4) * (kBM * 128) + (k % 4) * 32;
          tc_mma_f16(tmem_S, umma_smem_desc(aQ + off, 16, 1024), umma_smem_desc(aK + off, 16, 1024), kIdescS, k > 0 ? 1u : 0u);
        }
        tc_commit(s_full);
        if (!mbar_wait(p_ready, j & 1)) {
          report_status(p.status, kStatusWaitTmemFullTimeout);
          break;
        }
        if (!mbar_wait(v_full, j & 1)) {
          report_status(p.status, kStatusWaitFullTimeout);
          break;
        }
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < kBN / 16; ++k)
          tc_mma_f16_ts(tmem_O, tmem_S + k * 8, umma_smem_desc(aV + k * 2048, kBN * 128, 1024), kIdescO, (j > 0 || k > 0) ? 1u : 0u);
        tc_commit(o_done);
      }
    }
  } else {
    // Softmax and output: thread = one query row.
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const int qi = pos0 + r;
    const int first = qi / p.chunk * p.chunk;              // oldest key of this row
    const int last_first = (pos0 + n_rows - 1) / p.chunk * p.chunk;
    const uint32_t lane_off = static_cast<uint32_t>(quarter * 32) << 16;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < n_kv; ++j) {
      if (!mbar_wait(s_full, j & 1)) {
        report_status(p.status, kStatusWaitTmemFullTimeout);
        ok = false;
        break;
      }
      tc_fence_after();
      const int key0 = j0 + j * kBN;
      const bool masked = key0 + kBN - 1 > pos0 || key0 < last_first;
      const int lo = first - key0, hi = qi - key0;         // visible keys of the tile
      if constexpr (FREE) {
        if (j > 0 && !mbar_wait(o_done, (j - 1) & 1)) {    // P of the tile before has been read
          report_status(p.status, kStatusWaitTmemFullTimeout);
          ok = false;
          break;
        }
        tc_fence_after();
        uint32_t s[2][32];
        tmem_ld_32x32(tmem_S + lane_off, s[0]);
        tc_wait_ld();
#pragma unroll
        for (int c = 0; c < kBN / 32; ++c) {
          if (c + 1 < kBN / 32) tmem_ld_32x32(tmem_S + lane_off + (c + 1) * 32, s[(c + 1) & 1]);
          uint32_t w[16];
          if (masked) free_weights<true>(s[c & 1], p.sc, lo - c * 32, hi - c * 32, w, l);
          else free_weights<false>(s[c & 1], p.sc, 0, 0, w, l);
          tc_wait_ld();
          tmem_st_32x16(tmem_S + lane_off + c * 16, w);
        }
      } else {
        float mx = -INFINITY;
#pragma unroll 1
        for (int c = 0; c < kBN / 32; ++c) {
          uint32_t s[32];
          tmem_ld_32x32(tmem_S + lane_off + c * 32, s);
          tc_wait_ld();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int key = c * 32 + i;
            if (!masked || (key >= lo && key <= hi)) mx = fmaxf(mx, p.sc(__uint_as_float(s[i])));
          }
        }
        // a stale maximum is kept unless it grew by more than 2^8: weights stay bounded and O rarely needs rescaling
        float m_new = m, alpha = 1.f;
        if (mx > m + 8.f) {
          m_new = mx;
          alpha = m == -INFINITY ? 0.f : exp2f(m - m_new);
        }
        const bool need = j > 0 && alpha != 1.f;
        if (j > 0) {
          if (!mbar_wait(o_done, (j - 1) & 1)) {
            report_status(p.status, kStatusWaitTmemFullTimeout);
            ok = false;
            break;
          }
          tc_fence_after();
        }
        if (__any_sync(0xffffffffu, need)) {
#pragma unroll 1
          for (int c = 0; c < E / 16; ++c) {
            uint32_t o[16];
            tmem_ld_32x16(tmem_O + lane_off + c * 16, o);
            tc_wait_ld();
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st_32x16(tmem_O + lane_off + c * 16, o);
          }
        }
        l *= alpha;
        m = m_new;
        const float base = m == -INFINITY ? 0.f : m;
#pragma unroll 1
        for (int c = 0; c < kBN / 32; ++c) {
          uint32_t s[32], w[16];
          tmem_ld_32x32(tmem_S + lane_off + c * 32, s);
          tc_wait_ld();
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            float v[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int key = c * 32 + 2 * i + e;
              v[e] = !masked || (key >= lo && key <= hi) ? exp2f(p.sc(__uint_as_float(s[2 * i + e])) - base) : 0.f;
            }
            l += v[0] + v[1];
            w[i] = pack_bf16x2(v[0], v[1]);
          }
          tmem_st_32x16(tmem_S + lane_off + c * 16, w);
        }
      }
      tc_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    if (ok && mbar_wait(o_done, (n_kv - 1) & 1)) {
      tc_fence_after();
      const float inv = l > 0.f ? 1.f / l : 0.f;
      bf16* dst = p.out + (long long)(tile.x + r) * p.ldo + (long long)head * E;
#pragma unroll 1
      for (int c = 0; c < E / 32; ++c) {
        uint32_t o[32];
        tmem_ld_32x32(tmem_O + lane_off + c * 32, o);
        tc_wait_ld();
        if (r < n_rows) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            uint4 w;
            w.x = pack_bf16x2(__uint_as_float(o[i]) * inv, __uint_as_float(o[i + 1]) * inv);
            w.y = pack_bf16x2(__uint_as_float(o[i + 2]) * inv, __uint_as_float(o[i + 3]) * inv);
            w.z = pack_bf16x2(__uint_as_float(o[i + 4]) * inv, __uint_as_float(o[i + 5]) * inv);
            w.w = pack_bf16x2(__uint_as_float(o[i + 6]) * inv, __uint_as_float(o[i + 7]) * inv);
            *reinterpret_cast<uint4*>(dst + c * 32 + i) = w;
          }
        }
      }
    } else if (ok) {
      report_status(p.status, kStatusWaitTmemFullTimeout);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_S, kTmemCols);
  }
}

template <int D, int E>
void launch_prefill_t(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const ChunkPrefillParams& p, bool free_cap, int H, int n_tiles,
                      cudaStream_t s) {
  constexpr int smem = kBM * D * 2 + kBN * (D + E) * 2 + 64 + 1024;
  if (free_cap) {
    auto kernel = chunk_prefill_kernel<D, E, true>;
    AGRPO_SET_MAX_DYN_SMEM(kernel, smem, "chunk_prefill smem attr");
    launch_kernel(kernel, dim3(H, n_tiles), dim3(kThreads), smem, s, "chunk_prefill", tq, tk, tv, p);
  } else {
    auto kernel = chunk_prefill_kernel<D, E, false>;
    AGRPO_SET_MAX_DYN_SMEM(kernel, smem, "chunk_prefill smem attr");
    launch_kernel(kernel, dim3(H, n_tiles), dim3(kThreads), smem, s, "chunk_prefill", tq, tk, tv, p);
  }
}

// ================================================================================================
// Decode: CTA = (split, up to 16 query heads of one key head, sequence), four warps that take every fourth 16-token page of the
// part of the chunk that their split owns. Pages are requested before the step's projection is complete; then the CTA
// normalises and rotates its query heads into shared memory, and the split that owns the newest page also prepares the new key,
// writes it (and the value) to the cache and puts both into its copy of the page. ROWS: rows of the MMA that hold heads.
// ================================================================================================
constexpr int kWarps = 4;
constexpr int kStages = 2;
constexpr int kPage = 16;

template <int W>
__device__ __forceinline__ uint8_t* page_chunk(uint8_t* tile, int row, int chunk) {  // rows of W values, swizzled 16-byte chunks
  return tile + row * (W * 2) + ((chunk ^ (row & 7)) << 4);
}

__device__ __forceinline__ void norm_rotate(const QkRopeArgs& p, const bf16* src, const bf16* w, float inv, int i, const float* ct, const float* st, bf16* dst) {
  const int half = p.rot / 2;
  if (i < half) {
    const float a = ldf(src + i) * inv * ldf(w + i), b = ldf(src + half + i) * inv * ldf(w + half + i);
    const float c = ct[i], s = st[i];
    stf(dst + i, a * c - b * s);
    stf(dst + half + i, b * c + a * s);
  } else {
    stf(dst + half + i, ldf(src + half + i) * inv * ldf(w + half + i));
  }
}

template <int D, int E, int ROWS>
__global__ void __launch_bounds__(kWarps * 32, 3) chunk_decode_kernel(const ChunkDecodeArgs a, const CapScale sc) {
  constexpr int kTile = kPage * (D + E) * 2;
  constexpr int kQPitch = D + 8;
  extern __shared__ __align__(128) uint8_t cd_smem[];
  __shared__ __align__(16) bf16 sq[16 * kQPitch];
  __shared__ __align__(16) bf16 snew[D + E];
  __shared__ float sml[kWarps * ROWS * 2];
  __shared__ int s_last;
  const ChunkAttnArgs& at = a.at;
  const QkRopeArgs& qk = a.qk;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  const int b = blockIdx.z, split = blockIdx.x;
  const int grp = at.H / at.G, subs = (grp + 15) / 16;
  const int kvh = blockIdx.y / subs, e0 = (blockIdx.y % subs) * 16;
  const int nh = grp - e0 < 16 ? grp - e0 : 16;
  const int h0 = kvh * grp + e0;
  const int pos = at.seq_lens[b] - 1;
  if (pos < 0) return;
  if (pos >= qk.max_pos) {
    if (tid == 0) report_status(at.status, kStatusBadIndex);
    return;
  }
  const int lo = pos / at.chunk * at.chunk;
  const int page0 = lo / kPage, n_pages = pos / kPage + 1 - page0;
  const int p_begin = page0 + (int)((long long)n_pages * split / a.splits);
  const int p_end = page0 + (int)((long long)n_pages * (split + 1) / a.splits);
  const bool owner = p_begin < p_end && p_end == page0 + n_pages;
  const int* table = at.block_tables + (size_t)b * at.max_blocks;
  uint8_t* wbuf = cd_smem + warp * (kStages * kTile);

  auto physical = [&](int page) {
    int phys = table[page];
    if (phys < 0 || phys >= at.num_cache_blocks) {
      report_status(at.status, kStatusBadIndex);
      phys = 0;
    }
    return phys;
  };
  auto request = [&](int page, int stage) {
    const int phys = physical(page);
    const bf16* ks = reinterpret_cast<const bf16*>(at.k_cache) + ((size_t)phys * at.G + kvh) * kPage * D;
    const bf16* vs = reinterpret_cast<const bf16*>(at.v_cache) + ((size_t)phys * at.G + kvh) * kPage * E;
    uint8_t* kt = wbuf + stage * kTile;
    uint8_t* vt = kt + kPage * D * 2;
#pragma unroll
    for (int i = 0; i < D / 16; ++i) {
      const int idx = i * 32 + lane, row = idx / (D / 8), chunk = idx % (D / 8);
      cp_async16(page_chunk<D>(kt, row, chunk), ks + row * D + chunk * 8);
    }
#pragma unroll
    for (int i = 0; i < E / 16; ++i) {
      const int idx = i * 32 + lane, row = idx / (E / 8), chunk = idx % (E / 8);
      cp_async16(page_chunk<E>(vt, row, chunk), vs + row * E + chunk * 8);
    }
  };
  int my = p_begin + warp;
#pragma unroll
  for (int i = 0; i < kStages - 1; ++i) {
    if (my + i * kWarps < p_end) request(my + i * kWarps, i);
    cp_async_commit();
  }
  pdl_wait();
  pdl_launch();
  // ---- new token: query heads, and the key where this split owns its page ----
  {
    const bf16* u = reinterpret_cast<const bf16*>(qk.u) + (size_t)b * qk.ldu;
    const int half = qk.rot / 2, per = D - half;
    const float* ct = qk.cos_t + (size_t)pos * half;
    const float* st = qk.sin_t + (size_t)pos * half;
    const float iq = rsqrtf(sumsq_from_fixed(qk.ss_q[b]) / (float)(qk.H * qk.dim) + qk.eps);
    for (int i = tid; i < nh * per; i += kWarps * 32) {
      const int e = i / per;
      norm_rotate(qk, u + (size_t)(h0 + e) * D, reinterpret_cast<const bf16*>(qk.q_norm) + (size_t)(h0 + e) * D, iq, i % per, ct, st, sq + e * kQPitch);
    }
    for (int i = tid; i < (16 - nh) * (D / 2); i += kWarps * 32)
      *reinterpret_cast<uint32_t*>(sq + (nh + i / (D / 2)) * kQPitch + (i % (D / 2)) * 2) = 0u;
    if (owner) {
      const float ik = rsqrtf(sumsq_from_fixed(qk.ss_k[b]) / (float)(qk.G * qk.dim) + qk.eps);
      const bf16* kn = u + (size_t)(qk.H + kvh) * D;
      for (int i = tid; i < per; i += kWarps * 32)
        norm_rotate(qk, kn, reinterpret_cast<const bf16*>(qk.k_norm) + (size_t)kvh * D, ik, i, ct, st, snew);
      const bf16* vn = u + (size_t)(qk.H + qk.G) * D + (size_t)kvh * E;
      for (int i = tid; i < E; i += kWarps * 32) snew[D + i] = vn[i];
    }
  }
  __syncthreads();
  if (owner && warp == kWarps - 1) {
    const int phys = physical(pos / kPage);
    bf16* kd = reinterpret_cast<bf16*>(qk.k_cache) + (((size_t)phys * at.G + kvh) * kPage + pos % kPage) * D;
    bf16* vd = reinterpret_cast<bf16*>(qk.v_cache) + (((size_t)phys * at.G + kvh) * kPage + pos % kPage) * E;
    for (int i = lane; i < D / 8; i += 32) *reinterpret_cast<uint4*>(kd + i * 8) = *reinterpret_cast<const uint4*>(snew + i * 8);
    for (int i = lane; i < E / 8; i += 32) *reinterpret_cast<uint4*>(vd + i * 8) = *reinterpret_cast<const uint4*>(snew + D + i * 8);
  }
  uint32_t qa[D / 16][4];
#pragma unroll
  for (int kk = 0; kk < D / 16; ++kk) ldmatrix_x4(qa[kk], sq + (lane & 15) * kQPitch + kk * 16 + (lane >> 4) * 8);
  constexpr int kR = ROWS / 8;                // rows of heads per thread
  float o[E / 8][2 * kR];
#pragma unroll
  for (int n = 0; n < E / 8; ++n)
#pragma unroll
    for (int i = 0; i < 2 * kR; ++i) o[n][i] = 0.f;
  float m[kR], l[kR];
#pragma unroll
  for (int i = 0; i < kR; ++i) {
    m[i] = -INFINITY;
    l[i] = 0.f;
  }
  int stage = 0;
  for (; my < p_end; my += kWarps, stage = stage + 1 == kStages ? 0 : stage + 1) {
    const int nxt = my + (kStages - 1) * kWarps;
    if (nxt < p_end) request(nxt, stage == 0 ? kStages - 1 : stage - 1);
    cp_async_commit();
    cp_async_wait<kStages - 1>();
    __syncwarp();
    uint8_t* kt = wbuf + stage * kTile;
    uint8_t* vt = kt + kPage * D * 2;
    if (my == pos / kPage) {                  // the newest row is not in memory yet (or not seen here): put it into the copy
      const int row = pos % kPage;
      for (int i = lane; i < D / 8; i += 32) *reinterpret_cast<uint4*>(page_chunk<D>(kt, row, i)) = *reinterpret_cast<const uint4*>(snew + i * 8);
      for (int i = lane; i < E / 8; i += 32) *reinterpret_cast<uint4*>(page_chunk<E>(vt, row, i)) = *reinterpret_cast<const uint4*>(snew + D + i * 8);
      __syncwarp();
    }
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t kb[4];
      ldmatrix_x4(kb, page_chunk<D>(kt, (lane & 7) + ((lane >> 4) << 3), kk * 2 + ((lane >> 3) & 1)));
      mma_16816(s0, qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], kb[0], kb[1]);
      mma_16816(s1, qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], kb[2], kb[3]);
    }
    const int tok0 = my * kPage + (lane & 3) * 2;   // tokens {tok0, +1, +8, +9}
    uint32_t pa[4] = {0u, 0u, 0u, 0u};
    float alpha[kR];
#pragma unroll
    for (int rr = 0; rr < kR; ++rr) {
      float v[4] = {s0[2 * rr], s0[2 * rr + 1], s1[2 * rr], s1[2 * rr + 1]};
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int tok = tok0 + (i & 1) + (i >> 1) * 8;
        v[i] = tok >= lo && tok <= pos ? sc(v[i]) : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m_new = fmaxf(m[rr], mx);
      const float base = m_new == -INFINITY ? 0.f : m_new;
      alpha[rr] = m[rr] == -INFINITY ? 0.f : ex2(m[rr] - m_new);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[i] = ex2(v[i] - base);
        sum += v[i];
      }
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      l[rr] = l[rr] * alpha[rr] + sum;
      m[rr] = m_new;
      pa[rr] = pack_bf16x2(v[0], v[1]);
      pa[rr + 2] = pack_bf16x2(v[2], v[3]);
    }
#pragma unroll
    for (int n2 = 0; n2 < E / 16; ++n2) {
      uint32_t vb[4];
      ldmatrix_x4_trans(vb, page_chunk<E>(vt, (lane & 7) + (((lane >> 3) & 1) << 3), n2 * 2 + (lane >> 4)));
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        float c[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int rr = 0; rr < kR; ++rr) {
          c[2 * rr] = o[n2 * 2 + k][2 * rr] * alpha[rr];
          c[2 * rr + 1] = o[n2 * 2 + k][2 * rr + 1] * alpha[rr];
        }
        mma_16816(c, pa[0], pa[1], pa[2], pa[3], vb[2 * k], vb[2 * k + 1]);
#pragma unroll
        for (int i = 0; i < 2 * kR; ++i) o[n2 * 2 + k][i] = c[i];
      }
    }
    __syncwarp();
  }
  // ---- merge the warps, then the splits ----
  __syncthreads();
  float* mo = reinterpret_cast<float*>(cd_smem);   // [warps][ROWS][E]
#pragma unroll
  for (int rr = 0; rr < kR; ++rr) {
    const int g = (lane >> 2) + rr * 8;
#pragma unroll
    for (int n = 0; n < E / 8; ++n)
      *reinterpret_cast<float2*>(mo + (warp * ROWS + g) * E + n * 8 + (lane & 3) * 2) = make_float2(o[n][2 * rr], o[n][2 * rr + 1]);
    if ((lane & 3) == 0) {
      sml[(warp * ROWS + g) * 2] = m[rr];
      sml[(warp * ROWS + g) * 2 + 1] = l[rr];
    }
  }
  __syncthreads();
  bf16* out = reinterpret_cast<bf16*>(at.out) + (size_t)b * at.ldo;
  for (int idx = tid; idx < nh * E; idx += kWarps * 32) {
    const int g = idx / E, d = idx % E;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) M = fmaxf(M, sml[(w * ROWS + g) * 2]);
    float L = 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float mw = sml[(w * ROWS + g) * 2];
      const float wgt = mw == -INFINITY ? 0.f : ex2(mw - M);
      L += sml[(w * ROWS + g) * 2 + 1] * wgt;
      acc += mo[(w * ROWS + g) * E + d] * wgt;
    }
    if (a.splits == 1) {
      out[(size_t)(h0 + g) * E + d] = __float2bfloat16(L > 0.f ? acc / L : 0.f);
    } else {
      const size_t at_part = ((size_t)b * at.H + h0 + g) * a.splits + split;
      a.part_o[at_part * E + d] = acc;
      if (d == 0) {
        a.part_ml[at_part * 2] = M;
        a.part_ml[at_part * 2 + 1] = L;
      }
    }
  }
  if (a.splits == 1) return;
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    int* t = a.tickets + (size_t)b * at.H + h0;
    s_last = atomicAdd(t, 1) == a.splits - 1 ? 1 : 0;
    if (s_last) *t = 0;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  for (int idx = tid; idx < nh * (E / 4); idx += kWarps * 32) {
    const int g = idx / (E / 4), d = (idx % (E / 4)) * 4;
    const size_t base = ((size_t)b * at.H + h0 + g) * a.splits;
    float ms[8], ls[8], M = -INFINITY, L = 0.f;
    float4 os[8], acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < 8; ++j) {              // at most eight splits: all loads in flight before the first use
      const bool on = j < a.splits;
      const float2 ml = __ldcg(reinterpret_cast<const float2*>(a.part_ml + (base + (on ? j : 0)) * 2));
      ms[j] = on ? ml.x : -INFINITY;
      ls[j] = on ? ml.y : 0.f;
      os[j] = __ldcg(reinterpret_cast<const float4*>(a.part_o + (base + (on ? j : 0)) * E + d));
      M = fmaxf(M, ms[j]);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float w = ms[j] == -INFINITY ? 0.f : ex2(ms[j] - M);
      L += ls[j] * w;
      acc.x += os[j].x * w; acc.y += os[j].y * w; acc.z += os[j].z * w; acc.w += os[j].w * w;
    }
    const float inv = L > 0.f ? 1.f / L : 0.f;
    uint2 w;
    w.x = pack_bf16x2(acc.x * inv, acc.y * inv);
    w.y = pack_bf16x2(acc.z * inv, acc.w * inv);
    *reinterpret_cast<uint2*>(out + (size_t)(h0 + g) * E + d) = w;
  }
}

template <int D, int E, int ROWS>
void launch_decode_t(const ChunkDecodeArgs& a, cudaStream_t s) {
  constexpr int smem = kWarps * kStages * kPage * (D + E) * 2;
  static_assert(smem >= kWarps * ROWS * E * 4, "merge area");
  auto kernel = chunk_decode_kernel<D, E, ROWS>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, smem, "chunk_decode smem attr");
  AGRPO_PREFER_SMEM(kernel);
  const int grp = a.at.H / a.at.G;
  launch_kernel(kernel, dim3(a.splits, a.at.G * ((grp + 15) / 16), a.at.T), dim3(kWarps * 32), smem, s, "chunk_decode", a,
                cap_scale(a.at.scale, a.at.softcap));
}
template <int D, int E>
void launch_decode_rows(const ChunkDecodeArgs& a, cudaStream_t s) {
  if (a.at.H / a.at.G <= 8) launch_decode_t<D, E, 8>(a, s);
  else launch_decode_t<D, E, 16>(a, s);
}

}  // namespace

bool launch_chunk_attn_prefill(const ChunkAttnArgs& a, int q_cols, const int* tiles, int n_tiles, const int* pages, int n_pages, void* keys,
                               void* values, cudaStream_t s) {
  if ((a.D != 64 && a.D != 128) || (a.E != 64 && a.E != 128) || a.block_size != 16) return false;
  if (n_tiles == 0) return true;
  if (n_tiles > 65535) return false;
  launch_gather_pages(a.k_cache, pages, n_pages, a.block_tables, a.max_blocks, keys, a.G, a.D, a.num_cache_blocks, a.status, s);
  launch_gather_pages(a.v_cache, pages, n_pages, a.block_tables, a.max_blocks, values, a.G, a.E, a.num_cache_blocks, a.status, s);
  const CUtensorMap tq = make_tmap_2d(a.q, q_cols, a.T, a.ldq, 64, kBM);
  const CUtensorMap tk = make_tmap_2d(keys, a.G * a.D, (uint64_t)n_pages * 16, a.G * a.D, 64, kBN);
  const CUtensorMap tv = make_tmap_2d(values, a.G * a.E, (uint64_t)n_pages * 16, a.G * a.E, 64, kBN);
  ChunkPrefillParams p;
  p.tiles = reinterpret_cast<const int4*>(tiles);
  p.out = reinterpret_cast<bf16*>(a.out);
  p.ldo = a.ldo;
  p.group = a.H / a.G;
  p.chunk = a.chunk;
  p.sc = cap_scale(a.scale, a.softcap);
  p.status = a.status;
  const bool free_cap = a.softcap > 0.f && a.softcap <= kFreeCap;
  if (a.D == 128 && a.E == 128) launch_prefill_t<128, 128>(tq, tk, tv, p, free_cap, a.H, n_tiles, s);
  else if (a.D == 128) launch_prefill_t<128, 64>(tq, tk, tv, p, free_cap, a.H, n_tiles, s);
  else if (a.E == 128) launch_prefill_t<64, 128>(tq, tk, tv, p, free_cap, a.H, n_tiles, s);
  else launch_prefill_t<64, 64>(tq, tk, tv, p, free_cap, a.H, n_tiles, s);
  return true;
}

bool chunk_decode_serves(int H, int G, int D, int E) { return (D == 64 || D == 128) && (E == 64 || E == 128) && H % G == 0; }

void launch_chunk_attn_decode(const ChunkDecodeArgs& a, cudaStream_t s) {
  if (a.at.T == 0) return;
  if (a.at.D == 128 && a.at.E == 128) launch_decode_rows<128, 128>(a, s);
  else if (a.at.D == 128) launch_decode_rows<128, 64>(a, s);
  else if (a.at.E == 128) launch_decode_rows<64, 128>(a, s);
  else launch_decode_rows<64, 64>(a, s);
}

}  // namespace agrpo
