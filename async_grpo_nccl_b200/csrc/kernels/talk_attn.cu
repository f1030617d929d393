// Sliding-window attention with head mixing after the softmax ("talking heads") on the tensor cores, over paged keys that
// are also the values.
//
// Mixing makes output head h a combination over ALL heads g of softmax weights applied to h's own values,
//   out_h = sum_g talk[h, g] (P_g V_kv(h)) / l_g,
// and matrix products are linear, so the kernels never mix weights: they accumulate A[g, m] = P_g V_m for every query head
// g and key head m and combine those products at the end, in 32-bit. Scores never leave the chip and one pass over the keys
// is enough. With G key heads the price is (1 + G) / 2 times the products of unmixed attention in a prompt, and nothing in
// a decode step (the G products share the padded rows of one MMA).
//
// Scores are in log2 units: s = (q . k) * qscale[position] - bias[head][distance], both tables prepared by the caller.
#include <cuda_bf16.h>

#include "../common/ptx.cuh"
#include "../common/tensormap.h"
#include "../launchers.h"
#include "../launchers_layers.h"
#include "decode_attn.cuh"
#include "layer_ops.cuh"

namespace agrpo {

namespace {

typedef __nv_bfloat16 bf16;

// ================================================================================================
// Prompts: one CTA = 128 query rows of one head g, value heads [m0, m0 + mc). S (two buffers, so that the scores of tile
// j + 1 are computed while the softmax of tile j runs) and the mc accumulators fill tensor memory. Warp 0 loads key tiles
// page by page, warp 1 issues MMAs, warps 2-9 run the softmax: two threads per query row, 64 keys each. The key tile of
// a head serves as K-major operand of Q K^T and as MN-major operand of P V.
// ================================================================================================
constexpr int kPM = 128;
constexpr int kPN = 128;
constexpr int kPThreads = 320;
constexpr int kRingBytes = 192 * 1024;

struct TalkPrefillParams {
  const int4* tiles;       // {first row, rows, position of the first row, slot}
  const int* block_tables;
  int max_blocks;
  const float* bias;
  int bias_len;
  const float* qscale;
  int qscale_len;
  int window;
  bf16* acc;               // [T, H, G, D], normalised products
  int H, G, group, mc;     // mc = value heads per CTA
  int num_cache_blocks;
  int* status;
};

__device__ __forceinline__ void softmax_bar() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

template <int D>
__global__ void __launch_bounds__(kPThreads, 1)
talk_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const TalkPrefillParams p) {
  constexpr int kTile = kPM * D * 2;
  constexpr int kChunks = D / 64;
  constexpr uint32_t kIdescS = umma_idesc_bf16(kPM, kPN, 0, 0);
  constexpr uint32_t kIdescO = umma_idesc_bf16(kPM, D, 0, 1);
  extern __shared__ __align__(1024) uint8_t tp_smem[];
  uint8_t* sQ = tp_smem;
  uint8_t* sK = tp_smem + kTile;
  float* smax = reinterpret_cast<float*>(sK + kRingBytes);   // [2 parities][2 halves][128]
  uint64_t* bars = reinterpret_cast<uint64_t*>(smax + 512);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;      // [3]
  uint64_t* k_empty = bars + 4;     // [3]
  uint64_t* s_full = bars + 7;      // [2]
  uint64_t* p_ready = bars + 9;
  uint64_t* o_done = bars + 10;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 11);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.x;
  const int kv_own = head / p.group;
  const int m0 = blockIdx.y * p.mc;
  const int mc = p.G - m0 < p.mc ? p.G - m0 : p.mc;
  const int own_in = kv_own >= m0 && kv_own < m0 + mc ? kv_own - m0 : mc;  // place of the head's own keys in a stage
  const int n_t = own_in == mc ? mc + 1 : mc;
  const int stage_bytes = n_t * kTile;
  const int n_stages = kRingBytes / stage_bytes < 3 ? kRingBytes / stage_bytes : 3;
  const int4 tile = p.tiles[blockIdx.z];
  const int pos0 = tile.z, n_rows = tile.y;
  const int key_end = pos0 + n_rows;
  const int lo = pos0 - p.window + 1;
  const int j0 = lo > 0 ? (lo / 16) * 16 : 0;
  const int n_kv = (key_end - j0 + kPN - 1) / kPN;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 3; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
    }
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    mbar_init(p_ready, 8);
    mbar_init(o_done, 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_wait();
  pdl_launch();
  const uint32_t tmem = *tmem_slot;
  const uint32_t tmem_O = tmem + 256;

  if (warp == 0) {
    // ---------------- loads: lane b < 8 brings the b-th 16-token page of every tile ----------------
    if (lane == 0) {
      mbar_expect_tx(q_full, kTile);
#pragma unroll
      for (int c = 0; c < kChunks; ++c) tma_load_2d(sQ + c * (kPM * 128), &tmQ, q_full, head * D + c * 64, tile.x);
    }
    const int* table = p.block_tables + (size_t)tile.w * p.max_blocks;
    const int last_block = (key_end - 1) / 16;
    int stage = 0;
    uint32_t phase = 0;
    for (int j = 0; j < n_kv; ++j) {
      int phys = 0;
      if (lane < 8) {
        int bi = (j0 + j * kPN) / 16 + lane;
        bi = bi > last_block ? last_block : bi;  // past the end: any valid page, masked below
        phys = table[bi];
        if (phys < 0 || phys >= p.num_cache_blocks) {
          report_status(p.status, kStatusBadIndex);
          phys = 0;
        }
      }
      int good = 1;
      if (lane == 0) {
        if (j >= n_stages && !mbar_wait(&k_empty[stage], phase ^ 1)) {
          report_status(p.status, kStatusWaitEmptyTimeout);
          good = 0;
        }
        if (good) mbar_expect_tx(&k_full[stage], stage_bytes);
      }
      good = __shfl_sync(0xffffffffu, good, 0);
      if (!good) break;
      if (lane < 8) {
        uint8_t* dst = sK + stage * stage_bytes + lane * (16 * 128);
        for (int i = 0; i < n_t; ++i) {
          const int m = i < mc ? m0 + i : kv_own;
#pragma unroll
          for (int c = 0; c < kChunks; ++c)
            tma_load_2d(dst + i * kTile + c * (kPN * 128), &tmK, &k_full[stage], c * 64, (phys * p.G + m) * 16);
        }
      }
      if (++stage == n_stages) {
        stage = 0;
        phase ^= 1;
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (elect_one()) {
      const uint32_t aQ = smem_u32(sQ), aK = smem_u32(sK);
      auto scores = [&](int j, int stage) {
        const uint32_t kt = aK + stage * stage_bytes + own_in * kTile;
#pragma unroll
        for (int k = 0; k < D / 16; ++k) {
          const uint32_t off = (k / 4) * (kPM * 128) + (k % 4) * 32;
          tc_mma_f16(tmem + (j & 1) * 128, umma_smem_desc(aQ + off, 16, 1024), umma_smem_desc(kt + off, 16, 1024), kIdescS, k > 0 ? 1u : 0u);
        }
        tc_commit(&s_full[j & 1]);
      };
      bool ok = mbar_wait(q_full, 0) && mbar_wait(&k_full[0], 0);
      if (ok) {
        tc_fence_after();
        scores(0, 0);
      } else {
        report_status(p.status, kStatusWaitFullTimeout);
      }
      int stage = 0, nstage = n_stages > 1 ? 1 : 0;
      uint32_t nphase = n_stages > 1 ? 0 : 1;
      for (int j = 0; j < n_kv && ok; ++j) {
        if (j + 1 < n_kv) {
          // the buffer that the next scores go to holds the weights of tile j - 1 until their products are done
          if (j >= 1 && !mbar_wait(o_done, (j - 1) & 1)) {
            report_status(p.status, kStatusWaitTmemEmptyTimeout);
            break;
          }
          if (!mbar_wait(&k_full[nstage], nphase)) {
            report_status(p.status, kStatusWaitFullTimeout);
            break;
          }
          tc_fence_after();
          scores(j + 1, nstage);
        }
        if (!mbar_wait(p_ready, j & 1)) {
          report_status(p.status, kStatusWaitTmemFullTimeout);
          break;
        }
        tc_fence_after();
        for (int m = 0; m < mc; ++m) {
          const uint32_t vt = aK + stage * stage_bytes + m * kTile;
#pragma unroll
          for (int k = 0; k < kPN / 16; ++k)
            tc_mma_f16_ts(tmem_O + m * D, tmem + (j & 1) * 128 + k * 8, umma_smem_desc(vt + k * 2048, kPN * 128, 1024), kIdescO,
                          (j > 0 || k > 0) ? 1u : 0u);
        }
        tc_commit(&k_empty[stage]);
        tc_commit(o_done);
        stage = nstage;
        if (++nstage == n_stages) {
          nstage = 0;
          nphase ^= 1;
        }
      }
    }
  } else {
    // ---------------- softmax: thread = (query row, half of the tile's keys) ----------------
    const int quarter = warp & 3, half = (warp - 2) >> 2;
    const int r = quarter * 32 + lane;
    const int qi = pos0 + r;
    const uint32_t lane_off = static_cast<uint32_t>(quarter * 32) << 16;
    const float qs = p.qscale[qi < p.qscale_len ? qi : p.qscale_len - 1];
    const float* bias = p.bias + (size_t)head * p.bias_len;
    const int o_cols = mc * D / 2;            // accumulator columns that this half rescales and stores
    float m = -INFINITY, l = 0.f;
    bool ok = true;                           // after a failure the barriers are still met, nothing else is waited for
    for (int j = 0; j < n_kv; ++j) {
      if (ok && !mbar_wait(&s_full[j & 1], (j >> 1) & 1)) {
        report_status(p.status, kStatusWaitTmemFullTimeout);
        ok = false;
      }
      tc_fence_after();
      const uint32_t tS = tmem + (j & 1) * 128 + lane_off;
      const int tk = j0 + j * kPN;            // first key of the tile
      const int d0 = qi - (tk + half * 64);   // distance of this thread's first key
      uint32_t s0[32], s1[32];
      tmem_ld_32x32(tS + half * 64, s0);
      tmem_ld_32x32(tS + half * 64 + 32, s1);
      tc_wait_ld();
      float v[64];
      float mx = -INFINITY;
      const bool inside = tk + kPN - 1 <= pos0 && pos0 + kPM - 1 - tk < p.window && pos0 + kPM - 1 - tk < p.bias_len;
      if (inside) {
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          v[i] = fmaf(__uint_as_float(i < 32 ? s0[i & 31] : s1[i & 31]), qs, -__ldg(bias + d0 - i));
          mx = fmaxf(mx, v[i]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          const int d = d0 - i;
          const bool on = d >= 0 && d < p.window && d < p.bias_len;
          const float b = __ldg(bias + (on ? d : 0));
          v[i] = on ? fmaf(__uint_as_float(i < 32 ? s0[i & 31] : s1[i & 31]), qs, -b) : -INFINITY;
          mx = fmaxf(mx, v[i]);
        }
      }
      smax[((j & 1) * 2 + half) * 128 + r] = mx;
      tc_fence_before();
      softmax_bar();                          // both halves have read their scores: the weights may overwrite them
      tc_fence_after();
      mx = fmaxf(mx, smax[((j & 1) * 2 + (half ^ 1)) * 128 + r]);
      // keep a stale maximum unless it grew by more than 2^8: the weights stay bounded and O rarely needs rescaling
      float alpha = 1.f;
      if (mx > m + 8.f || m == -INFINITY) {
        if (m != -INFINITY) alpha = exp2f(m - mx);  // nothing has been accumulated before the first visible key
        m = mx;
      }
      const float base = m == -INFINITY ? 0.f : m;
      if (__any_sync(0xffffffffu, alpha != 1.f)) {
        if (ok && !mbar_wait(o_done, (j - 1) & 1)) {
          report_status(p.status, kStatusWaitTmemFullTimeout);
          ok = false;
        }
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c < o_cols; c += 32) {
          const uint32_t a = tmem_O + lane_off + half * o_cols + c;
          uint32_t o[32];
          tmem_ld_32x32(a, o);
          tc_wait_ld();
          uint32_t x0[16], x1[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            x0[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            x1[i] = __float_as_uint(__uint_as_float(o[16 + i]) * alpha);
          }
          tmem_st_32x16(a, x0);
          tmem_st_32x16(a + 16, x1);
        }
        l *= alpha;
      }
      uint32_t w0[16], w1[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const float a = exp2f(v[2 * i] - base), b = exp2f(v[2 * i + 1] - base);
        const float c = exp2f(v[32 + 2 * i] - base), d = exp2f(v[32 + 2 * i + 1] - base);
        l += (a + b) + (c + d);
        w0[i] = pack_bf16x2(a, b);
        w1[i] = pack_bf16x2(c, d);
      }
      tmem_st_32x16(tS + half * 32, w0);
      tmem_st_32x16(tS + half * 32 + 16, w1);
      tc_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    // the two halves of a row add up their sums
    softmax_bar();
    smax[half * 128 + r] = l;
    softmax_bar();
    l += smax[(half ^ 1) * 128 + r];
    if (ok && !mbar_wait(o_done, (n_kv - 1) & 1)) {
      report_status(p.status, kStatusWaitTmemFullTimeout);
      ok = false;
    }
    tc_fence_after();
    const float inv = l > 0.f ? 1.f / l : 0.f;
    bf16* dst = p.acc + (((size_t)(tile.x + r) * p.H + head) * p.G + m0) * D + half * o_cols;
#pragma unroll 1
    for (int c = 0; c < o_cols; c += 32) {
      uint32_t o[32];
      tmem_ld_32x32(tmem_O + lane_off + half * o_cols + c, o);
      tc_wait_ld();
      if (ok && r < n_rows) {
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          uint4 w;
          w.x = pack_bf16x2(__uint_as_float(o[i]) * inv, __uint_as_float(o[i + 1]) * inv);
          w.y = pack_bf16x2(__uint_as_float(o[i + 2]) * inv, __uint_as_float(o[i + 3]) * inv);
          w.z = pack_bf16x2(__uint_as_float(o[i + 4]) * inv, __uint_as_float(o[i + 5]) * inv);
          w.w = pack_bf16x2(__uint_as_float(o[i + 6]) * inv, __uint_as_float(o[i + 7]) * inv);
          *reinterpret_cast<uint4*>(dst + c + i) = w;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// out[t, h] = sigmoid(gate[t, h]) * sum_g talk[h, g] acc[t, g, kv(h)]. Thread = four dims of one key head; the heads of its
// group are accumulated eight at a time.
constexpr int kMixThreads = 256;
constexpr int kMixTokens = 8;

__global__ void __launch_bounds__(kMixThreads)
talk_mix_gate_kernel(const bf16* __restrict__ acc, const bf16* __restrict__ talk, const bf16* __restrict__ gate, long long ldg,
                     bf16* __restrict__ out, long long ldo, int T, int H, int G, int D) {
  extern __shared__ __align__(16) float mix_t[];  // [G][H (g)][gp]: talk transposed, heads of a group contiguous
  pdl_wait();
  pdl_launch();
  const int grp = H / G, gp = (grp + 7) & ~7;
  for (int i = threadIdx.x; i < G * H * gp; i += kMixThreads) {
    const int e = i % gp, g = (i / gp) % H, m = i / (gp * H);
    mix_t[i] = e < grp ? (talk != nullptr ? ldf(talk + (size_t)(m * grp + e) * H + g) : (g == m * grp + e ? 1.f : 0.f)) : 0.f;
  }
  __syncthreads();
  const int per_tok = G * D / 4;
  const int t0 = blockIdx.x * kMixTokens;
  const int n = (T - t0 < kMixTokens ? T - t0 : kMixTokens) * per_tok;
  for (int i = threadIdx.x; i < n; i += kMixThreads) {
    const int t = t0 + i / per_tok, c = (i % per_tok) * 4, m = c / D, d = c % D;
    const bf16* src = acc + (size_t)t * H * G * D + c;
    for (int e0 = 0; e0 < grp; e0 += 8) {
      float o[8][4];
#pragma unroll
      for (int e = 0; e < 8; ++e)
#pragma unroll
        for (int k = 0; k < 4; ++k) o[e][k] = 0.f;
#pragma unroll 4
      for (int g = 0; g < H; ++g) {
        const uint2 w = *reinterpret_cast<const uint2*>(src + (size_t)g * G * D);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
        const float4* tr = reinterpret_cast<const float4*>(mix_t + (m * H + g) * gp + e0);
        const float4 ta = tr[0], tb = tr[1];
        const float tt[8] = {ta.x, ta.y, ta.z, ta.w, tb.x, tb.y, tb.z, tb.w};
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          o[e][0] = fmaf(tt[e], a.x, o[e][0]);
          o[e][1] = fmaf(tt[e], a.y, o[e][1]);
          o[e][2] = fmaf(tt[e], b.x, o[e][2]);
          o[e][3] = fmaf(tt[e], b.y, o[e][3]);
        }
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        if (e0 + e >= grp) break;
        const int h = m * grp + e0 + e;
        if (gate != nullptr) {
          const uint2 w = *reinterpret_cast<const uint2*>(gate + (size_t)t * ldg + h * D + d);
          const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
          const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
          o[e][0] *= sigmoid_f32(a.x);
          o[e][1] *= sigmoid_f32(a.y);
          o[e][2] *= sigmoid_f32(b.x);
          o[e][3] *= sigmoid_f32(b.y);
        }
        uint2 w;
        w.x = pack_bf16x2(o[e][0], o[e][1]);
        w.y = pack_bf16x2(o[e][2], o[e][3]);
        *reinterpret_cast<uint2*>(out + (size_t)t * ldo + h * D + d) = w;
      }
    }
  }
}

template <int D>
void launch_prefill_t(const CUtensorMap& tq, const CUtensorMap& tk, const TalkPrefillParams& p, int n_tiles, int chunks, cudaStream_t s) {
  constexpr int smem = kPM * D * 2 + kRingBytes + 512 * 4 + 128;
  auto kernel = talk_prefill_kernel<D>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, smem, "talk_prefill smem attr");
  launch_kernel(kernel, dim3(p.H, chunks, n_tiles), dim3(kPThreads), smem, s, "talk_prefill", tq, tk, p);
}

// ================================================================================================
// Decode: CTA = (split, sequence), 8 warps, all heads. The prologue convolves the new token's q (every split) and k (the
// split that owns the newest token, which also writes the key page and the ring). Per tile of 64 keys: warp w scores its 8
// keys against all heads, the CTA agrees on the row maxima, the weights meet in shared memory, and warp w accumulates its
// share of the G * D value columns for all heads. The last split of a sequence to finish merges, mixes, gates and stores.
// ================================================================================================
constexpr int kDT = 64;         // keys per tile
constexpr int kDThreads = 256;
constexpr int kPPitch = kDT + 8;

template <int D, int MT>
struct DecSmem {
  static constexpr int kRowBytes = D * 2;
  static constexpr int kQ = MT * 16 * kRowBytes;
  static constexpr int kP = MT * 16 * kPPitch * 2;
  static constexpr int kMax = MT * 16 * 8 * 4;
};

template <int D>
__device__ __forceinline__ uint8_t* sw_chunk(uint8_t* base, int row, int chunk) {  // 16-byte chunks, conflict-free for ldmatrix
  return base + row * (D * 2) + ((chunk ^ (row & 7)) << 4);
}

// eight channels of the convolution of the token at `pos` (its own value in u, older ones in the ring)
__device__ __forceinline__ void conv8(const TalkDecodeArgs& a, int b, int pos, int C, int c, float (&acc)[8]) {
  const bf16* w = reinterpret_cast<const bf16*>(a.conv_w) + (size_t)c * a.taps;
  const bf16* ring = reinterpret_cast<const bf16*>(a.ring) + (size_t)b * a.ring_pitch;
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.f;
  for (int back = a.taps - 1; back >= 0; --back) {
    if (pos - back < 0) continue;
    float v[8];
    ld8(back == 0 ? reinterpret_cast<const bf16*>(a.u) + (size_t)b * a.ldu + c : ring + (size_t)((pos - back) % a.ring_len) * C + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = fmaf(ldf(w + i * a.taps + a.taps - 1 - back), v[i], acc[i]);
  }
}

template <int D, int MT, int NTW>
__global__ void __launch_bounds__(kDThreads) talk_decode_kernel(const TalkDecodeArgs a, const int n_stages) {
  extern __shared__ __align__(1024) uint8_t td_smem[];
  __shared__ int s_last;
  const WindowAttnArgs& p = a.at;
  const int H = p.H, G = p.G, grp = H / G, GD = G * D;
  const int stage_bytes = kDT * GD * 2;
  uint8_t* sKV = td_smem;                                        // [stages][G][64][D], later the fp32 products [H][G * D]
  uint8_t* sQ = sKV + n_stages * stage_bytes;
  uint8_t* sP = sQ + DecSmem<D, MT>::kQ;
  float* sMax = reinterpret_cast<float*>(sP + DecSmem<D, MT>::kP);   // [MT * 16][8]
  bf16* sKnew = reinterpret_cast<bf16*>(reinterpret_cast<uint8_t*>(sMax) + DecSmem<D, MT>::kMax);  // [G * D]
  float* sTalk = reinterpret_cast<float*>(sKnew + GD);           // [H][H]
  const int split = blockIdx.x, b = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_wait();
  pdl_launch();
  const int pos = p.seq_lens[b] - 1;
  if (pos < 0) return;
  const int C = H * D + GD;
  const int lo = pos - p.window + 1 > 0 ? pos - p.window + 1 : 0;
  const int n_tiles = (pos - lo) / kDT + 1;
  const int t_begin = (int)((long long)n_tiles * split / a.splits), t_end = (int)((long long)n_tiles * (split + 1) / a.splits);
  const bool newest = split == a.splits - 1;
  const int* table = p.block_tables + (size_t)b * p.max_blocks;
  const bf16* cache = reinterpret_cast<const bf16*>(p.k_cache);

  // Pages of the next tile to load, one per lane (a tile of 64 keys touches at most five): looked up one tile ahead, so that
  // no copy waits for its table entry.
  int page = 0;
  auto fetch_pages = [&](int t) {
    const int bi = (lo + t * kDT) / 16 + lane;
    if (t < t_end && lane < 5 && bi <= pos / 16) {
      page = table[bi];
      if (page < 0 || page >= p.num_cache_blocks) {
        report_status(p.status, kStatusBadIndex);
        page = 0;
      }
    }
  };
  auto load_tile = [&](int t, int stage) {
    constexpr int kRowChunks = D / 8;
    uint8_t* dst = sKV + stage * stage_bytes;
    const int jt = lo + t * kDT, b0 = jt / 16;
    const int n = kDT * G * kRowChunks;                      // a multiple of the CTA's threads: warps stay whole
#pragma unroll 4
    for (int i = tid; i < n; i += kDThreads) {
      const int ch = i % kRowChunks, row = i / kRowChunks;   // row = m * 64 + key
      const int m = row / kDT;
      int j = jt + row % kDT;
      const bool on = j < pos;                               // the newest key comes from sKnew, later ones are masked
      const int blk = __shfl_sync(0xffffffffu, page, on ? j / 16 - b0 : 0);
      j = on ? j : 0;
      if (on) cp_async16(sw_chunk<D>(dst, row, ch), cache + (((size_t)blk * G + m) * 16 + j % 16) * D + ch * 8);
      else if (row % kDT != pos - jt) *reinterpret_cast<uint4*>(sw_chunk<D>(dst, row, ch)) = make_uint4(0u, 0u, 0u, 0u);
    }
    fetch_pages(t + 1);
  };
  // loads first: they do not depend on the new token
  fetch_pages(t_begin);
  for (int i = 0; i < n_stages - 1; ++i) {
    if (t_begin + i < t_end) load_tile(t_begin + i, i);
    cp_async_commit();
  }
  for (int i = tid; i < MT * 16 * (D / 8); i += kDThreads) {
    const int row = i / (D / 8), ch = i % (D / 8);
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (row < H) conv8(a, b, pos, C, row * D + ch * 8, v);
    st8(reinterpret_cast<bf16*>(sw_chunk<D>(sQ, row, ch)), v);
  }
  if (newest) {
    int blk = table[pos / 16];
    if (blk < 0 || blk >= p.num_cache_blocks) {
      report_status(p.status, kStatusBadIndex);
      blk = 0;
    }
    for (int i = tid; i < GD / 8; i += kDThreads) {
      const int c = i * 8, m = c / D, d = c % D;
      float v[8];
      conv8(a, b, pos, C, H * D + c, v);
      st8(sKnew + c, v);
      st8(reinterpret_cast<bf16*>(a.k_cache) + (((size_t)blk * G + m) * 16 + pos % 16) * D + d, v);
    }
    if (a.taps > 1) {  // nobody reads this ring entry before the next token
      const bf16* u = reinterpret_cast<const bf16*>(a.u) + (size_t)b * a.ldu;
      bf16* ring = reinterpret_cast<bf16*>(a.ring) + (size_t)b * a.ring_pitch + (size_t)(pos % a.ring_len) * C;
      for (int i = tid * 8; i < C; i += kDThreads * 8) *reinterpret_cast<uint4*>(ring + i) = *reinterpret_cast<const uint4*>(u + i);
    }
  }
  if (p.talk != nullptr)
    for (int i = tid; i < H * H; i += kDThreads) sTalk[i] = ldf(reinterpret_cast<const bf16*>(p.talk) + i);

  const float qs = p.qscale[pos < p.qscale_len ? pos : p.qscale_len - 1];
  const int npw = (GD / 8 + 7) / 8;              // 8-wide value-column tiles per warp
  const int nt0 = warp * npw;
  const int r0 = lane >> 2, cq = (lane & 3) * 2;
  float acc[MT][NTW][4];
  float mrow[MT][2], lrow[MT][2];
#pragma unroll
  for (int t = 0; t < MT; ++t) {
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) acc[t][i][k] = 0.f;
    mrow[t][0] = mrow[t][1] = -INFINITY;
    lrow[t][0] = lrow[t][1] = 0.f;
  }
  __syncthreads();  // q, the new key and the mixing matrix are in shared memory
  int stage = 0;
  for (int t = t_begin; t < t_end; ++t) {
    if (n_stages == 1) {
      __syncthreads();
      load_tile(t, 0);
      cp_async_commit();
      cp_async_wait<0>();
    } else if (n_stages == 2) {
      cp_async_wait<0>();
    } else {
      cp_async_wait<1>();
    }
    uint8_t* kt = sKV + stage * stage_bytes;
    const int j0 = lo + t * kDT;
    if (newest && t == t_end - 1) {
      const int key = pos - j0;
      for (int i = tid; i < GD / 8; i += kDThreads) {
        const int m = i / (D / 8), ch = i % (D / 8);
        *reinterpret_cast<uint4*>(sw_chunk<D>(kt, m * kDT + key, ch)) = *reinterpret_cast<const uint4*>(sKnew + i * 8);
      }
    }
    __syncthreads();  // the tile is complete; everybody is done with the stage that is loaded next
    if (n_stages > 1) {
      const int nxt = t + n_stages - 1;
      if (nxt < t_end) load_tile(nxt, stage == 0 ? n_stages - 1 : stage - 1);
      cp_async_commit();
    }
    // ---- scores of keys [8 warp, 8 warp + 8) for all heads ----
    float s[MT][4], bv[MT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {  // distance biases, on their way while the MMAs run
        const int h = mt * 16 + r0 + (e >> 1) * 8;
        const int d = pos - (j0 + warp * 8 + cq + (e & 1));
        const bool on = h < H && d >= 0 && d < p.window && d < p.bias_len;
        bv[mt][e] = on ? __ldg(p.bias + (size_t)h * p.bias_len + d) : INFINITY;
      }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      s[mt][0] = s[mt][1] = s[mt][2] = s[mt][3] = 0.f;
      const int h_lo = mt * 16, h_hi = (mt * 16 + 16 < H ? mt * 16 + 16 : H) - 1;
      const int ka = (h_lo + r0) / grp, kb = (h_lo + r0 + 8) / grp;   // key heads of this thread's two rows
      for (int m = h_lo / grp; m <= h_hi / grp && h_hi >= h_lo; ++m) {
        const bool ua = ka == m, ub = kb == m;
#pragma unroll
        for (int kk = 0; kk < D / 32; ++kk) {
          uint32_t kf[4];  // two k-steps of 16 for 8 keys
          ldmatrix_x4(kf, sw_chunk<D>(kt, m * kDT + warp * 8 + (lane & 7), kk * 4 + (lane >> 3)));
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            uint32_t qf[4];
            ldmatrix_x4(qf, sw_chunk<D>(sQ, h_lo + (lane & 7) + ((lane >> 3) & 1) * 8, (kk * 2 + half) * 2 + (lane >> 4)));
            mma_16816(s[mt], ua ? qf[0] : 0u, ub ? qf[1] : 0u, ua ? qf[2] : 0u, ub ? qf[3] : 0u, kf[half * 2], kf[half * 2 + 1]);
          }
        }
      }
      // scale, distance bias, mask; row maxima over this warp's keys
#pragma unroll
      for (int e = 0; e < 4; ++e) s[mt][e] = fmaf(s[mt][e], qs, -bv[mt][e]);  // masked: minus infinity
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        float mx = fmaxf(s[mt][2 * q], s[mt][2 * q + 1]);
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        if ((lane & 3) == 0) sMax[(h_lo + r0 + q * 8) * 8 + warp] = mx;
      }
    }
    __syncthreads();
    // ---- weights ----
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      float al[2];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int row = mt * 16 + r0 + q * 8;
        const float4 x = *reinterpret_cast<const float4*>(sMax + row * 8), y = *reinterpret_cast<const float4*>(sMax + row * 8 + 4);
        const float mx = fmaxf(fmaxf(fmaxf(x.x, x.y), fmaxf(x.z, x.w)), fmaxf(fmaxf(y.x, y.y), fmaxf(y.z, y.w)));
        const float mn = fmaxf(mrow[mt][q], mx);
        al[q] = mrow[mt][q] == -INFINITY ? 0.f : exp2f(mrow[mt][q] - mn);
        mrow[mt][q] = mn;
        const float base = mn == -INFINITY ? 0.f : mn;
        const float p0 = exp2f(s[mt][2 * q] - base), p1 = exp2f(s[mt][2 * q + 1] - base);
        lrow[mt][q] = lrow[mt][q] * al[q] + p0 + p1;
        *reinterpret_cast<uint32_t*>(sP + (row * kPPitch + warp * 8 + cq) * 2) = pack_bf16x2(p0, p1);
      }
#pragma unroll
      for (int i = 0; i < NTW; ++i) {
        acc[mt][i][0] *= al[0];
        acc[mt][i][1] *= al[0];
        acc[mt][i][2] *= al[1];
        acc[mt][i][3] *= al[1];
      }
    }
    __syncthreads();
    // ---- products: all heads x this warp's value columns ----
#pragma unroll
    for (int kk = 0; kk < kDT / 16; ++kk) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
        ldmatrix_x4(pf[mt], sP + ((mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kPPitch + kk * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
      for (int i = 0; i < NTW; i += (NTW > 1 ? 2 : 1)) {
        if (i < npw && nt0 + i < GD / 8) {
          // x4: two neighbouring column tiles (the second one may belong to the next warp; it is then not used)
          const int n1 = nt0 + i;
          const int n2 = n1 + 1 < GD / 8 ? n1 + 1 : n1;
          const int nn = (lane >> 4) ? n2 : n1;
          const int m = nn / (D / 8), ch = nn % (D / 8);
          uint32_t vf[4];
          ldmatrix_x4_trans(vf, sw_chunk<D>(kt, m * kDT + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, ch));
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma_16816(acc[mt][i], pf[mt][0], pf[mt][1], pf[mt][2], pf[mt][3], vf[0], vf[1]);
            if constexpr (NTW > 1) {
              if (i + 1 < npw) mma_16816(acc[mt][i + 1], pf[mt][0], pf[mt][1], pf[mt][2], pf[mt][3], vf[2], vf[3]);
            }
          }
        }
      }
    }
    stage = stage + 1 == n_stages ? 0 : stage + 1;
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- row sums over the warps ----
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      float l = lrow[mt][q];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      if ((lane & 3) == 0) sMax[(mt * 16 + r0 + q * 8) * 8 + warp] = l;
    }
  __syncthreads();
  float* prod = reinterpret_cast<float*>(sKV);   // [H][G * D]
  const size_t part = ((size_t)b * a.splits + split) * H;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int h = mt * 16 + r0 + q * 8;
      if (h >= H) continue;
      float l = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) l += sMax[h * 8 + w];
      const float inv = a.splits == 1 ? (l > 0.f ? 1.f / l : 0.f) : 1.f;
      float* dst = a.splits == 1 ? prod + (size_t)h * GD : a.part_o + (part + h) * GD;
#pragma unroll
      for (int i = 0; i < NTW; ++i)
        if (i < npw && nt0 + i < GD / 8)
          *reinterpret_cast<float2*>(dst + (nt0 + i) * 8 + cq) = make_float2(acc[mt][i][2 * q] * inv, acc[mt][i][2 * q + 1] * inv);
      if (a.splits > 1 && warp == 0 && (lane & 3) == 0)
        *reinterpret_cast<float2*>(a.part_ml + (part + h) * 2) = make_float2(mrow[mt][q], l);
    }
  if (a.splits > 1) {
    __threadfence();
    __syncthreads();
    if (tid == 0) {
      const int ticket = atomicAdd(a.tickets + b, 1);
      s_last = ticket == a.splits - 1;
      if (s_last) a.tickets[b] = 0;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    float* wgt = sMax;  // [H][splits] merge weights, splits <= 8
    for (int h = tid; h < H; h += kDThreads) {
      const size_t base = (size_t)b * a.splits * H + h;
      float M = -INFINITY, L = 0.f;
      for (int s = 0; s < a.splits; ++s) M = fmaxf(M, __ldcg(a.part_ml + (base + (size_t)s * H) * 2));
      for (int s = 0; s < a.splits; ++s) {
        const float2 ml = __ldcg(reinterpret_cast<const float2*>(a.part_ml + (base + (size_t)s * H) * 2));
        const float w = ml.x == -INFINITY ? 0.f : exp2f(ml.x - M);
        wgt[h * 8 + s] = w;
        L += ml.y * w;
      }
      for (int s = 0; s < a.splits; ++s) wgt[h * 8 + s] *= L > 0.f ? 1.f / L : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < H * GD / 4; i += kDThreads) {
      const int h = i / (GD / 4);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < 8; ++s) {
        if (s < a.splits) {
          const float4 x = __ldcg(reinterpret_cast<const float4*>(a.part_o + ((size_t)b * a.splits + s) * H * GD) + i);
          const float w = wgt[h * 8 + s];
          o.x = fmaf(x.x, w, o.x); o.y = fmaf(x.y, w, o.y); o.z = fmaf(x.z, w, o.z); o.w = fmaf(x.w, w, o.w);
        }
      }
      reinterpret_cast<float4*>(prod)[i] = o;
    }
  }
  __syncthreads();
  // ---- mix across heads, gate, store ----
  const bf16* gate = p.gate != nullptr ? reinterpret_cast<const bf16*>(p.gate) + (size_t)b * p.ldg : nullptr;
  bf16* out = reinterpret_cast<bf16*>(p.out) + (size_t)b * p.ldo;
  for (int i = tid; i < H * D / 2; i += kDThreads) {
    const int h = i / (D / 2), d = (i % (D / 2)) * 2;
    const float* src = prod + (h / grp) * D + d;
    float x = 0.f, y = 0.f;
    if (p.talk != nullptr) {
      for (int g = 0; g < H; ++g) {
        const float2 v = *reinterpret_cast<const float2*>(src + (size_t)g * GD);
        const float w = sTalk[h * H + g];
        x = fmaf(w, v.x, x);
        y = fmaf(w, v.y, y);
      }
    } else {
      x = src[(size_t)h * GD];
      y = src[(size_t)h * GD + 1];
    }
    if (gate != nullptr) {
      x *= sigmoid_f32(ldf(gate + h * D + d));
      y *= sigmoid_f32(ldf(gate + h * D + d + 1));
    }
    *reinterpret_cast<uint32_t*>(out + h * D + d) = pack_bf16x2(x, y);
  }
}

struct DecPlan {
  int mt, ntw, stages;
  size_t smem;
};
// picks the template and the number of stages; mt = 0: not served
DecPlan plan_decode_kernel(int H, int G, int D) {
  DecPlan d{0, 0, 0, 0};
  if ((D != 64 && D != 128) || H > 64 || H % G != 0) return d;
  const int mt = H <= 16 ? 1 : (H <= 32 ? 2 : 4);
  const int npw = (G * D / 8 + 7) / 8;
  int ntw = 1;
  while (ntw < npw) ntw *= 2;
  if (ntw > 16 || mt * ntw > 32) return d;
  const size_t stage = (size_t)kDT * G * D * 2;
  const size_t fixed = (size_t)mt * 16 * D * 2 + (size_t)mt * 16 * kPPitch * 2 + (size_t)mt * 16 * 32 + (size_t)G * D * 2 + (size_t)H * H * 4;
  const size_t prod = (size_t)H * G * D * 4;
  int st = 3;
  while (st > 1 && st * stage + fixed > (size_t)110 * 1024) --st;  // two CTAs per SM while that leaves two stages
  if (st < 2) {
    st = 2;
    if (st * stage + fixed > (size_t)224 * 1024) st = 1;
  }
  if (st * stage < prod) return d;
  if (st * stage + fixed > (size_t)224 * 1024) return d;
  d.mt = mt; d.ntw = ntw; d.stages = st; d.smem = st * stage + fixed;
  return d;
}

template <int D, int MT, int NTW>
void launch_decode_t(const TalkDecodeArgs& a, const DecPlan& d, cudaStream_t s) {
  auto kernel = talk_decode_kernel<D, MT, NTW>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, 226 * 1024, "talk_decode smem attr");
  AGRPO_PREFER_SMEM(kernel);
  launch_kernel(kernel, dim3(a.splits, a.at.T), dim3(kDThreads), d.smem, s, "talk_decode", a, d.stages);
}
template <int D, int MT>
void launch_decode_n(const TalkDecodeArgs& a, const DecPlan& d, cudaStream_t s) {
  if (d.ntw == 1) return launch_decode_t<D, MT, 1>(a, d, s);
  if (d.ntw == 2) return launch_decode_t<D, MT, 2>(a, d, s);
  if (d.ntw == 4) return launch_decode_t<D, MT, 4>(a, d, s);
  if (d.ntw == 8) return launch_decode_t<D, MT, 8>(a, d, s);
  if constexpr (MT <= 2) {
    if (d.ntw == 16) return launch_decode_t<D, MT, 16>(a, d, s);
  }
  throw std::runtime_error("talk_decode: shape not served");
}

}  // namespace

bool launch_talk_attn_prefill(const WindowAttnArgs& a, const int* tiles, int n_tiles, void* acc, cudaStream_t s) {
  if ((a.D != 64 && a.D != 128) || a.block_size != 16 || a.H % a.G != 0) return false;
  const int grp8 = (a.H / a.G + 7) & ~7;
  const size_t mix_smem = (size_t)a.G * a.H * grp8 * 4;
  if (mix_smem > 200 * 1024) return false;
  if (a.T == 0 || n_tiles == 0) return true;
  const int mc_max = 256 / a.D;
  const int chunks = (a.G + mc_max - 1) / mc_max;
  const CUtensorMap tq = make_tmap_2d(a.q, (uint64_t)a.H * a.D, a.T, a.ldq, 64, kPM);
  const CUtensorMap tk = make_tmap_2d(a.k_cache, a.D, (uint64_t)a.num_cache_blocks * a.G * 16, a.D, 64, 16);
  TalkPrefillParams p;
  p.tiles = reinterpret_cast<const int4*>(tiles);
  p.block_tables = a.block_tables;
  p.max_blocks = a.max_blocks;
  p.bias = a.bias;
  p.bias_len = a.bias_len;
  p.qscale = a.qscale;
  p.qscale_len = a.qscale_len;
  p.window = a.window;
  p.acc = reinterpret_cast<bf16*>(acc);
  p.H = a.H;
  p.G = a.G;
  p.group = a.H / a.G;
  p.mc = (a.G + chunks - 1) / chunks;
  p.num_cache_blocks = a.num_cache_blocks;
  p.status = a.status;
  if (a.D == 128) launch_prefill_t<128>(tq, tk, p, n_tiles, chunks, s);
  else launch_prefill_t<64>(tq, tk, p, n_tiles, chunks, s);
  AGRPO_SET_MAX_DYN_SMEM(talk_mix_gate_kernel, 200 * 1024, "talk_mix smem attr");
  launch_kernel(talk_mix_gate_kernel, dim3((a.T + kMixTokens - 1) / kMixTokens), dim3(kMixThreads), mix_smem, s, "talk_mix_gate",
                (const bf16*)acc, (const bf16*)a.talk, (const bf16*)a.gate, a.ldg, (bf16*)a.out, a.ldo, a.T, a.H, a.G, a.D);
  return true;
}

bool talk_decode_supported(int H, int G, int D) { return plan_decode_kernel(H, G, D).mt > 0; }

void launch_talk_attn_decode(const TalkDecodeArgs& a, cudaStream_t s) {
  const DecPlan d = plan_decode_kernel(a.at.H, a.at.G, a.at.D);
  if (d.mt == 0 || a.at.block_size != 16 || a.splits < 1 || a.splits > 8) throw std::runtime_error("talk_decode: shape not served");
  if (a.at.T == 0) return;
  if (a.at.D == 128) {
    if (d.mt == 1) launch_decode_n<128, 1>(a, d, s);
    else if (d.mt == 2) launch_decode_n<128, 2>(a, d, s);
    else launch_decode_n<128, 4>(a, d, s);
  } else {
    if (d.mt == 1) launch_decode_n<64, 1>(a, d, s);
    else if (d.mt == 2) launch_decode_n<64, 2>(a, d, s);
    else launch_decode_n<64, 4>(a, d, s);
  }
}

}  // namespace agrpo
