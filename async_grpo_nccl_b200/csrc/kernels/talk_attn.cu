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
#include "../launchers_hybrid.h"
#include "../launchers_layers.h"
#include "decode_attn.cuh"
#include "layer_ops.cuh"

namespace agrpo {

namespace {

typedef __nv_bfloat16 bf16;

// ================================================================================================
// Prompts: one CTA = 128 query rows of one head g, value heads [m0, m0 + mc). S (two buffers, so that the scores of tile
// j + 1 are computed while the softmax of tile j runs) and the mc accumulators fill tensor memory. The keys that a step can
// see are first gathered from their pages into one matrix (a TMA request per 16-token page would be the bottleneck). Warp 0
// loads key tiles into a ring of slots, one slot per key head of a tile, warp 1 issues MMAs, warps 2-17 run the softmax in two groups that take alternating tiles (one group's loads
// and maxima overlap the other's exponentials); in a group two threads share a query row, 64 keys each. The reference maximum
// of a row is handed from tile to tile through shared memory, so that all weights of a row are on one scale. The key tile of a
// head serves as K-major operand of Q K^T and as MN-major operand of P V.
// ================================================================================================
constexpr int kPM = 128;
constexpr int kPN = 128;
constexpr int kPKeys = 64;                            // keys per thread and tile
constexpr int kPThreads = 64 + 4 * kPM;
constexpr int kRingBytes = 192 * 1024;
constexpr int kMaxSlots = 12;

struct TalkPrefillParams {
  const int4* tiles;       // {first row, rows, position of the first row, row of position 0 among the gathered keys}
  const float* bias;
  int bias_len;
  const float* qscale;
  int qscale_len;
  int window;
  bf16* acc;               // [T, H, G, D], normalised products
  int H, G, group, mc;     // mc = value heads per CTA
  int* status;
};

__device__ __forceinline__ void softmax_group_bar(int group) { asm volatile("bar.sync %0, 256;" ::"r"(group + 1) : "memory"); }
__device__ __forceinline__ void softmax_all_bar() { asm volatile("bar.sync 3, 512;" ::: "memory"); }

template <int D>
__global__ void __launch_bounds__(kPThreads, 1)
talk_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const TalkPrefillParams p) {
  constexpr int kTile = kPM * D * 2;
  constexpr int kChunks = D / 64;
  constexpr int kSlots = kRingBytes / kTile;
  constexpr uint32_t kIdescS = umma_idesc_bf16(kPM, kPN, 0, 0);
  constexpr uint32_t kIdescO = umma_idesc_bf16(kPM, D, 0, 1);
  extern __shared__ __align__(1024) uint8_t tp_smem[];
  uint8_t* sQ = tp_smem;
  uint8_t* sK = tp_smem + kTile;
  float* smax = reinterpret_cast<float*>(sK + kRingBytes);   // 2 KB: row maxima [2 groups][2 turns][2 halves][128] as bf16, at the end sums
  bf16* smax16 = reinterpret_cast<bf16*>(smax);
  bf16* sref = reinterpret_cast<bf16*>(smax + 512);          // [2][128] reference maximum after the latest even / odd tile
  uint64_t* bars = reinterpret_cast<uint64_t*>(sref + 256);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 1;      // [2]
  uint64_t* p_ready = bars + 3;     // [2]
  uint64_t* ref_set = bars + 5;     // [2]
  // [2], even and odd tiles: a thread may look for tile j's products while those of tile j - 1 are still running, which one
  // barrier's parity could not tell from finished
  uint64_t* o_done = bars + 7;
  uint64_t* k_full = bars + 9;      // [kSlots]
  uint64_t* k_empty = k_full + kMaxSlots;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(k_empty + kMaxSlots);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.x;
  const int kv_own = head / p.group;
  const int m0 = blockIdx.y * p.mc;
  const int mc = p.G - m0 < p.mc ? p.G - m0 : p.mc;
  // a tile takes n_t slots: [own keys, when they are not among the value heads], value heads m0 ...
  const int extra = kv_own >= m0 && kv_own < m0 + mc ? 0 : 1;
  const int own_slot = extra ? 0 : kv_own - m0;
  const int n_t = mc + extra;
  const int4 tile = p.tiles[blockIdx.z];
  const int pos0 = tile.z, n_rows = tile.y;
  const int key_end = pos0 + n_rows;
  const int lo = pos0 - p.window + 1;
  const int j0 = lo > 0 ? (lo / 16) * 16 : 0;
  const int n_kv = (key_end - j0 + kPN - 1) / kPN;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < kSlots; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
    }
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&p_ready[i], 8);
      mbar_init(&ref_set[i], 8);
    }
    mbar_init(&o_done[0], 1);
    mbar_init(&o_done[1], 1);
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
    // ---------------- loads ----------------
    if (elect_one()) {
      mbar_expect_tx(q_full, kTile);
#pragma unroll
      for (int c = 0; c < kChunks; ++c) tma_load_2d(sQ + c * (kPM * 128), &tmQ, q_full, head * D + c * 64, tile.x);
      int slot = 0;
      uint32_t phase = 1;
      bool ok = true;
      for (int j = 0; j < n_kv && ok; ++j) {
        const int row = tile.w + j0 + j * kPN;   // rows past the gathered keys read as zero, other segments' rows are masked
        for (int k = 0; k < n_t; ++k) {
          if (!mbar_wait(&k_empty[slot], phase)) {
            report_status(p.status, kStatusWaitEmptyTimeout);
            ok = false;
            break;
          }
          const int m = extra ? (k == 0 ? kv_own : m0 + k - 1) : m0 + k;
          mbar_expect_tx(&k_full[slot], kTile);
#pragma unroll
          for (int c = 0; c < kChunks; ++c) tma_load_2d(sK + slot * kTile + c * (kPN * 128), &tmK, &k_full[slot], m * D + c * 64, row);
          if (++slot == kSlots) {
            slot = 0;
            phase ^= 1;
          }
        }
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (elect_one()) {
      const uint32_t aQ = smem_u32(sQ), aK = smem_u32(sK);
      auto wait_slot = [&](int idx) { return mbar_wait(&k_full[idx % kSlots], (idx / kSlots) & 1); };
      auto scores = [&](int j) {
        const int slot = (j * n_t + own_slot) % kSlots;
        const uint32_t kt = aK + slot * kTile;
#pragma unroll
        for (int k = 0; k < D / 16; ++k) {
          const uint32_t off = (k / 4) * (kPM * 128) + (k % 4) * 32;
          tc_mma_f16(tmem + (j & 1) * 128, umma_smem_desc(aQ + off, 16, 1024), umma_smem_desc(kt + off, 16, 1024), kIdescS, k > 0 ? 1u : 0u);
        }
        if (extra) tc_commit(&k_empty[slot]);   // these keys are not read as values
        tc_commit(&s_full[j & 1]);
      };
      bool ok = mbar_wait(q_full, 0) && wait_slot(own_slot);
      if (ok) {
        tc_fence_after();
        scores(0);
      } else {
        report_status(p.status, kStatusWaitFullTimeout);
      }
      for (int j = 0; j < n_kv && ok; ++j) {
        if (j + 1 < n_kv) {
          // the buffer that the next scores go to holds the weights of tile j - 1 until their products are done
          if (j >= 1 && !mbar_wait(&o_done[(j - 1) & 1], ((j - 1) >> 1) & 1)) {
            report_status(p.status, kStatusWaitTmemEmptyTimeout);
            break;
          }
          if (!wait_slot((j + 1) * n_t + own_slot)) {
            report_status(p.status, kStatusWaitFullTimeout);
            break;
          }
          tc_fence_after();
          scores(j + 1);
        }
        if (!mbar_wait(&p_ready[j & 1], (j >> 1) & 1)) {
          report_status(p.status, kStatusWaitTmemFullTimeout);
          break;
        }
        for (int m = 0; m < mc && ok; ++m) {
          const int idx = j * n_t + extra + m;
          ok = wait_slot(idx);
          tc_fence_after();
          const uint32_t vt = aK + (idx % kSlots) * kTile;
          if (ok) {
#pragma unroll
            for (int k = 0; k < kPN / 16; ++k)
              tc_mma_f16_ts(tmem_O + m * D, tmem + (j & 1) * 128 + k * 8, umma_smem_desc(vt + k * 2048, kPN * 128, 1024), kIdescO,
                            (j > 0 || k > 0) ? 1u : 0u);
            tc_commit(&k_empty[idx % kSlots]);
          }
        }
        if (!ok) {
          report_status(p.status, kStatusWaitFullTimeout);
          break;
        }
        tc_commit(&o_done[j & 1]);
      }
    }
  } else {
    // ---------------- softmax: thread = (query row, half of the keys of every second tile) ----------------
    const int group = (warp - 2) >> 3, half = ((warp - 2) >> 2) & 1, quarter = warp & 3;
    const int part = group * 2 + half;
    const int r = quarter * 32 + lane;
    const int qi = pos0 + r;
    const uint32_t lane_off = static_cast<uint32_t>(quarter * 32) << 16;
    const float qs = p.qscale[qi < p.qscale_len ? qi : p.qscale_len - 1];
    const float* bias = p.bias + (size_t)head * p.bias_len;
    const int h_cols = mc * D / 2;            // accumulator columns that this thread rescales
    const uint32_t tS = tmem + group * 128 + lane_off;
    float m = -INFINITY, l = 0.f;             // reference maximum of this group's latest tile, sum of its weights on that scale
    bool ok = true;                           // after a failure the barriers are still met, nothing else is waited for
    for (int j = group; j < n_kv; j += 2) {
      const int tk = j0 + j * kPN;            // first key of the tile
      const int d0 = qi - (tk + half * kPKeys);  // distance of this thread's first key
      const bool inside = tk + kPN - 1 <= pos0 && pos0 + kPM - 1 - tk < p.window && pos0 + kPM - 1 - tk < p.bias_len;
      if (ok && !mbar_wait(&s_full[group], (j >> 1) & 1)) {
        report_status(p.status, kStatusWaitTmemFullTimeout);
        ok = false;
      }
      tc_fence_after();
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      float v[kPKeys];
      // small pieces: a spill would cost an L2 round trip next to this much shared memory
      if (inside) {
#pragma unroll
        for (int c = 0; c < kPKeys; c += 8) {
          uint32_t s0[8];
          tmem_ld_32x8(tS + half * kPKeys + c, s0);
          float b[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) b[i] = __ldg(bias + d0 - c - i);
          tc_wait_ld();
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            v[c + i] = fmaf(__uint_as_float(s0[i]), qs, -b[i]);
            mx4[i & 3] = fmaxf(mx4[i & 3], v[c + i]);
          }
        }
      } else {
#pragma unroll
        for (int c = 0; c < kPKeys; c += 8) {
          uint32_t s0[8];
          tmem_ld_32x8(tS + half * kPKeys + c, s0);
          tc_wait_ld();
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const int d = d0 - c - i;
            const float b = d >= 0 && d < p.window && d < p.bias_len ? __ldg(bias + d) : INFINITY;
            v[c + i] = fmaf(__uint_as_float(s0[i]), qs, -b);  // masked keys: minus infinity
            mx4[i & 3] = fmaxf(mx4[i & 3], v[c + i]);
          }
        }
      }
      // the maximum is only a reference point: kept in bf16, the same rounded value for all threads of a row
      bf16* mine = smax16 + (group * 2 + ((j >> 1) & 1)) * 256;
      mine[half * 128 + r] = __float2bfloat16(fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])));
      tc_fence_before();
      softmax_group_bar(group);               // both halves have read their scores: the weights may overwrite them
      tc_fence_after();
      const float mx = fmaxf(__bfloat162float(mine[r]), __bfloat162float(mine[128 + r]));
      float m_prev = -INFINITY;               // scale of what is accumulated so far
      if (j > 0) {
        if (ok && !mbar_wait(&ref_set[group ^ 1], ((j - 1) >> 1) & 1)) {
          report_status(p.status, kStatusWaitTmemFullTimeout);
          ok = false;
        }
        m_prev = __bfloat162float(sref[(group ^ 1) * 128 + r]);
      }
      // keep a stale maximum unless it grew by more than 2^8: the weights stay bounded and O rarely needs rescaling
      const float m_new = (mx > m_prev + 8.f || m_prev == -INFINITY) ? mx : m_prev;
      if (half == 0) sref[group * 128 + r] = __float2bfloat16(m_new);
      __syncwarp();
      if (lane == 0) mbar_arrive(&ref_set[group]);
      const float alpha = m_prev == -INFINITY ? 1.f : exp2f(m_prev - m_new);  // nothing is accumulated before the first visible key
      if (__any_sync(0xffffffffu, alpha != 1.f)) {
        if (ok && !mbar_wait(&o_done[(j - 1) & 1], ((j - 1) >> 1) & 1)) {
          report_status(p.status, kStatusWaitTmemFullTimeout);
          ok = false;
        }
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c < h_cols; c += 16) {
          const uint32_t ta = tmem_O + lane_off + half * h_cols + c;
          uint32_t o[16];
          tmem_ld_32x16(ta, o);
          tc_wait_ld();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
          tmem_st_32x16(ta, o);
        }
      }
      if (m != m_new) l *= m == -INFINITY ? 0.f : exp2f(m - m_new);
      m = m_new;
      const float base = m == -INFINITY ? 0.f : m;
      float l0 = 0.f, l1 = 0.f;
#pragma unroll
      for (int c = 0; c < kPKeys; c += 32) {
        uint32_t w[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float a = exp2f(v[c + 2 * i] - base), b = exp2f(v[c + 2 * i + 1] - base);
          l0 += a;
          l1 += b;
          w[i] = pack_bf16x2(a, b);
        }
        tmem_st_32x16(tS + half * (kPKeys / 2) + c / 2, w);
      }
      l += l0 + l1;
      tc_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_ready[group]);
    }
    // the four threads of a row add up their sums on the scale of the last tile
    const int last = (n_kv - 1) & 1;
    if (ok && !mbar_wait(&ref_set[last], ((n_kv - 1) >> 1) & 1)) {
      report_status(p.status, kStatusWaitTmemFullTimeout);
      ok = false;
    }
    const float m_end = __bfloat162float(sref[last * 128 + r]);
    if (m != m_end) l *= m == -INFINITY ? 0.f : exp2f(m - m_end);
    softmax_all_bar();
    smax[part * 128 + r] = l;
    softmax_all_bar();
    l = (smax[r] + smax[128 + r]) + (smax[256 + r] + smax[384 + r]);
    if (ok && !mbar_wait(&o_done[last], ((n_kv - 1) >> 1) & 1)) {
      report_status(p.status, kStatusWaitTmemFullTimeout);
      ok = false;
    }
    tc_fence_after();
    const float inv = l > 0.f ? 1.f / l : 0.f;
    const int o_cols = mc * D / 4;
    bf16* dst = p.acc + (((size_t)(tile.x + r) * p.H + head) * p.G + m0) * D + part * o_cols;
#pragma unroll 1
    for (int c = 0; c < o_cols; c += 16) {
      uint32_t o[16];
      tmem_ld_32x16(tmem_O + lane_off + part * o_cols + c, o);
      tc_wait_ld();
      if (ok && r < n_rows) {
#pragma unroll
        for (int i = 0; i < 16; i += 8) {
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

// Brings the pages that a step can see into one matrix [rows, G * D]: CTA = page, 16 rows of the matrix.
__global__ void __launch_bounds__(128)
gather_keys_kernel(const bf16* __restrict__ cache, const int2* __restrict__ pages, const int* __restrict__ block_tables, int max_blocks,
                   bf16* __restrict__ keys, int G, int D, int num_cache_blocks, int* status) {
  const int2 pg = pages[blockIdx.x];  // {slot, page of the sequence}
  const int blk = block_tables[(size_t)pg.x * max_blocks + pg.y];
  if (blk < 0 || blk >= num_cache_blocks) {
    if (threadIdx.x == 0) report_status(status, kStatusBadIndex);
    return;
  }
  const int per_row = D / 8;
  const uint4* src = reinterpret_cast<const uint4*>(cache + (size_t)blk * G * 16 * D);
  uint4* dst = reinterpret_cast<uint4*>(keys + (size_t)blockIdx.x * 16 * G * D);
#pragma unroll 4
  for (int i = threadIdx.x; i < G * 16 * per_row; i += 128) {
    const int c = i % per_row, r = (i / per_row) % 16, m = i / (per_row * 16);
    dst[(r * G + m) * per_row + c] = src[i];
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
  constexpr int smem = kPM * D * 2 + kRingBytes + 512 * 4 + 256 * 2 + (9 + 2 * kMaxSlots) * 8 + 16;
  auto kernel = talk_prefill_kernel<D>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, smem, "talk_prefill smem attr");
  launch_kernel(kernel, dim3(p.H, chunks, n_tiles), dim3(kPThreads), smem, s, "talk_prefill", tq, tk, p);
}

// ================================================================================================
// Decode: CTA = (split, sequence), all heads: 8 warps per MTW row tiles of 16 heads; with one group of warps a further warp
// loads, with two (where it would cost the others registers) the first warp does. The prologue convolves the new token's q (every split) and k (the
// split that owns the newest token, which also writes the key page and the ring). Key tiles of 64 tokens arrive by TMA, page
// by page, from before the new token's projections are complete. Per tile: a warp scores its 8 keys against its heads, the
// CTA agrees on the row maxima, the weights meet in shared memory, and the warp accumulates its share of the G * D value
// columns for its heads. The last split of a sequence to finish merges, mixes, gates and stores.
// ================================================================================================
constexpr int kDT = 64;         // keys per tile
constexpr int kPPitch = kDT + 8;

template <int D, int MT>
struct DecSmem {
  static constexpr int kQ = MT * 16 * D * 2;
  static constexpr int kP = MT * 16 * kPPitch * 2;
  static constexpr int kMax = MT * 16 * 8 * 4;
};

// Rows of 64 channels (128 bytes), 16-byte chunk c of row r stored at c ^ (r & 7): the layout of a TMA box with 128-byte swizzle.
__device__ __forceinline__ uint32_t sw_off(int row, int chunk) { return row * 128 + ((chunk ^ (row & 7)) << 4); }

// eight channels of the convolution of the token at `pos` (its own value in u, older ones in the ring); weights [taps, C]
__device__ __forceinline__ void conv8(const TalkDecodeArgs& a, int b, int pos, int C, int c, float (&acc)[8]) {
  const bf16* w = reinterpret_cast<const bf16*>(a.conv_w) + c;
  const bf16* ring = reinterpret_cast<const bf16*>(a.ring) + (size_t)b * a.ring_pitch + c;
  const bf16* u = reinterpret_cast<const bf16*>(a.u) + (size_t)b * a.ldu + c;
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.f;
  int slot = pos % a.ring_len;
#pragma unroll 4
  for (int back = 0; back < a.taps; ++back) {
    if (pos - back >= 0) {
      float v[8], x[8];
      ld8(back == 0 ? u : ring + (size_t)slot * C, v);
      ld8(w + (size_t)(a.taps - 1 - back) * C, x);
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i] = fmaf(x[i], v[i], acc[i]);
    }
    slot = slot == 0 ? a.ring_len - 1 : slot - 1;
  }
}

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}

template <int N>
__device__ __forceinline__ void compute_bar() { asm volatile("bar.sync 1, %0;" ::"n"(N) : "memory"); }

// MW groups of 8 warps, MTW row tiles of 16 heads per warp, up to NTW 8-wide value-column tiles per warp
template <int D, int MW, int MTW, int NTW>
__global__ void __launch_bounds__(MW == 1 ? 288 : 512, (MW == 1 && NTW <= 4) ? 2 : 1)
talk_decode_kernel(const __grid_constant__ CUtensorMap tmK, const TalkDecodeArgs a, const int n_stages) {
  constexpr int MT = MW * MTW;
  constexpr int kDThreads = MW * 256;                            // computing threads
  constexpr int kPl = D / 64;                                    // planes of 64 channels
  constexpr bool kQReg = MTW == 1 && NTW <= 8;                   // query fragments stay in registers
  extern __shared__ __align__(1024) uint8_t td_smem[];
  const WindowAttnArgs& p = a.at;
  const int H = p.H, G = p.G, grp = H / G, GD = G * D;
  const int stage_bytes = kDT * GD * 2;
  uint8_t* sKV = td_smem;                                        // [stages][G][planes][64][128 B], later the fp32 products [H][G * D]
  uint8_t* sQ = sKV + n_stages * stage_bytes;                    // [MT][planes][16][128 B]
  uint8_t* sP = sQ + DecSmem<D, MT>::kQ;
  float* sMax = reinterpret_cast<float*>(sP + DecSmem<D, MT>::kP);   // [MT * 16][8]
  bf16* sKnew = reinterpret_cast<bf16*>(reinterpret_cast<uint8_t*>(sMax) + DecSmem<D, MT>::kMax);  // [G * D]
  float* sTalk = reinterpret_cast<float*>(sKnew + GD);           // [H][H]
  uint64_t* full = reinterpret_cast<uint64_t*>(sTalk + ((H * H + 1) & ~1));  // [4]
  uint64_t* empty = full + 4;                                    // [4]
  int* s_last = reinterpret_cast<int*>(empty + 4);
  const int split = blockIdx.x, b = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  // Lengths, tables and the keys of earlier tokens were complete before the kernel ahead of this one started.
  const int pos = p.seq_lens[b] - 1;
  if (pos < 0) {
    pdl_wait();
    pdl_launch();
    return;
  }
  const int C = H * D + GD;
  const int lo = pos - p.window + 1 > 0 ? pos - p.window + 1 : 0;
  const int jb = (lo / 16) * 16;
  const int n_tiles = (pos - jb) / kDT + 1;
  const int t_begin = (int)((long long)n_tiles * split / a.splits), t_end = (int)((long long)n_tiles * (split + 1) / a.splits);
  const bool newest = split == a.splits - 1;
  const int* table = p.block_tables + (size_t)b * p.max_blocks;

  if (tid == 0) {
    for (int i = 0; i < 4; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], MW * 8);
    }
    fence_mbar_init();
  }
  __syncthreads();
  // ---- loads: lane -> page (lane & 3) of a tile, looked up one tile ahead ----
  auto page_of = [&](int t) {
    const int bi = (jb + t * kDT) / 16 + (lane & 3);
    return t < t_end ? table[bi > pos / 16 ? pos / 16 : bi] : 0;  // past the end: any valid page, masked
  };
  int next_page = 0;
  auto issue_tile = [&](int page, int st) {
    uint8_t* dst = sKV + st * stage_bytes + (lane & 3) * (16 * 128);
    for (int i = lane >> 2; i < G * kPl; i += 8)
      tma_load_2d(dst + i * (kDT * 128), &tmK, &full[st], (i % kPl) * 64, (page * G + i / kPl) * 16);
  };
  auto load_tile = [&](int t, int st) {
    int page = next_page;
    next_page = page_of(t + 1);
    if (page < 0 || page >= p.num_cache_blocks) {
      report_status(p.status, kStatusBadIndex);
      page = 0;
    }
    if (lane == 0) mbar_expect_tx(&full[st], stage_bytes);
    __syncwarp();
    issue_tile(page, st);
  };
  if (MW == 1 && warp == 8) {
    int st = 0;
    uint32_t ph = 1;
    int next = t_begin < t_end ? page_of(t_begin) : 0;
    for (int t = t_begin; t < t_end; ++t) {
      int page = next;
      if (t + 1 < t_end) next = page_of(t + 1);
      if (page < 0 || page >= p.num_cache_blocks) {
        report_status(p.status, kStatusBadIndex);
        page = 0;
      }
      int good = 1;
      if (lane == 0) {
        if (!mbar_wait(&empty[st], ph)) {
          report_status(p.status, kStatusWaitEmptyTimeout);
          good = 0;
        } else {
          mbar_expect_tx(&full[st], stage_bytes);
        }
      }
      if (!__shfl_sync(0xffffffffu, good, 0)) break;
      issue_tile(page, st);
      if (++st == n_stages) {
        st = 0;
        ph ^= 1;
      }
    }
    pdl_wait();
    return;
  }
  if (MW == 2 && warp == 0) {
    next_page = page_of(t_begin);
    for (int i = 0; i < (n_stages > 1 ? n_stages - 1 : 1); ++i)
      if (t_begin + i < t_end) load_tile(t_begin + i, i);
  }
  if (p.talk != nullptr)
    for (int i = tid; i < H * H; i += kDThreads) sTalk[i] = ldf(reinterpret_cast<const bf16*>(p.talk) + i);
  pdl_wait();
  pdl_launch();
  for (int i = tid; i < MT * 16 * (D / 8); i += kDThreads) {
    const int row = i / (D / 8), ch = i % (D / 8);
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (row < H) conv8(a, b, pos, C, row * D + ch * 8, v);
    st8(reinterpret_cast<bf16*>(sQ + ((row >> 4) * kPl + (ch >> 3)) * 2048 + sw_off(row & 15, ch & 7)), v);
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

  const float qs = p.qscale[pos < p.qscale_len ? pos : p.qscale_len - 1];
  const int cw = warp & 7, mt0 = (warp >> 3) * MTW;  // warp within its group, first row tile
  const int nt0 = cw * NTW;                      // first of this warp's 8-wide value-column tiles
  const int n_cols = GD / 8;
  const int r0 = lane >> 2, cq = (lane & 3) * 2;
  // fragment addresses that do not change from tile to tile (inside a stage)
  const uint32_t k_off = sw_off(cw * 8 + (lane & 7), lane >> 3);                       // keys: chunks 0-3; chunks 4-7 at ^ 64
  const uint32_t q_off = smem_u32(sQ) + mt0 * kPl * 2048 + sw_off((lane & 7) + ((lane >> 3) & 1) * 8, lane >> 4);  // queries: k-step s at ^ (s * 32)
  const uint32_t p_off = smem_u32(sP) + ((mt0 * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kPPitch + (lane >> 4) * 8) * 2;
  constexpr int kPairs = NTW / 2;
  // value columns, two neighbouring 8-wide tiles per ldmatrix: pair i at (+ (i >> 2) planes) ^ (i & 3) * 32; few pairs keep
  // their addresses in registers
  constexpr bool kVReg = NTW <= 4;
  const uint32_t v_off = (nt0 >> 3) * (kDT * 128) + sw_off((lane & 7) + ((lane >> 3) & 1) * 8, (nt0 & 7) + (lane >> 4));
  uint32_t v_pair[kVReg ? kPairs : 1];
#pragma unroll
  for (int i = 0; i < (kVReg ? kPairs : 1); ++i) v_pair[i] = v_off ^ (i * 32);
  const float* bias_row[MTW][2];                  // rows past the last head read the last head's biases; they are never stored
  int key_head[MTW][2];
#pragma unroll
  for (int mt = 0; mt < MTW; ++mt)
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      int h = (mt0 + mt) * 16 + r0 + q * 8;
      h = h < H ? h : H - 1;
      bias_row[mt][q] = p.bias + (size_t)h * p.bias_len;
      key_head[mt][q] = h / grp;
    }
  int m_lo[MTW], m_hi[MTW];                      // key heads that a row tile reads
#pragma unroll
  for (int mt = 0; mt < MTW; ++mt) {
    const int h0 = (mt0 + mt) * 16, h1 = (h0 + 16 < H ? h0 + 16 : H) - 1;
    m_lo[mt] = h0 / grp;
    m_hi[mt] = h0 < H ? h1 / grp : -1;
  }
  float acc[MTW][NTW][4];
  float mrow[MTW][2], lrow[MTW][2];
#pragma unroll
  for (int t = 0; t < MTW; ++t) {
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) acc[t][i][k] = 0.f;
    mrow[t][0] = mrow[t][1] = -INFINITY;
    lrow[t][0] = lrow[t][1] = 0.f;
  }
  compute_bar<kDThreads>();  // q, the new key and the mixing matrix are in shared memory
  uint32_t qf[kQReg ? D / 16 : 1][4];
  if constexpr (kQReg) {
#pragma unroll
    for (int k = 0; k < D / 16; ++k) ldsm4(qf[k], (q_off + (k >> 2) * 2048) ^ ((k & 3) * 32));
  }
  int stage = 0;
  uint32_t phase = 0;
  bool ok = true;
  for (int t = t_begin; t < t_end; ++t) {
    const int j0 = jb + t * kDT;
    const bool inside = j0 >= lo && j0 + kDT - 1 <= pos && pos - j0 < p.bias_len;
    float bv[MTW][4];                             // distance biases, on their way while the tile arrives
    {
      const int d = pos - (j0 + cw * 8 + cq);
#pragma unroll
      for (int mt = 0; mt < MTW; ++mt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int de = d - (e & 1);
          if (inside) bv[mt][e] = __ldg(bias_row[mt][e >> 1] + de);
          else bv[mt][e] = de >= 0 && de < p.window && de < p.bias_len ? __ldg(bias_row[mt][e >> 1] + de) : INFINITY;
        }
    }
    if (ok && !mbar_wait(&full[stage], phase)) {
      report_status(p.status, kStatusWaitFullTimeout);
      ok = false;
    }
    uint8_t* kt = sKV + stage * stage_bytes;
    const uint32_t kts = smem_u32(kt);
    if (newest && t == t_end - 1) {
      const int key = pos - j0;
      for (int i = tid; i < GD / 8; i += kDThreads) {
        const int m = i / (D / 8), ch = i % (D / 8);
        *reinterpret_cast<uint4*>(kt + (m * kPl + (ch >> 3)) * (kDT * 128) + sw_off(key, ch & 7)) = *reinterpret_cast<const uint4*>(sKnew + i * 8);
      }
      compute_bar<kDThreads>();
    }
    // ---- scores of keys [8 warp, 8 warp + 8) for all heads ----
    float s[MTW][4];
#pragma unroll
    for (int mt = 0; mt < MTW; ++mt) {
      s[mt][0] = s[mt][1] = s[mt][2] = s[mt][3] = 0.f;
      for (int m = m_lo[mt]; m <= m_hi[mt]; ++m) {
        float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int pl = 0; pl < kPl; ++pl) {
          const uint32_t ka = kts + (m * kPl + pl) * (kDT * 128) + k_off;
          uint32_t k0[4], k1[4];
          ldsm4(k0, ka);
          ldsm4(k1, ka ^ 64);
          if constexpr (kQReg) {
            mma_16816(c0, qf[pl * 4][0], qf[pl * 4][1], qf[pl * 4][2], qf[pl * 4][3], k0[0], k0[1]);
            mma_16816(c1, qf[pl * 4 + 1][0], qf[pl * 4 + 1][1], qf[pl * 4 + 1][2], qf[pl * 4 + 1][3], k0[2], k0[3]);
            mma_16816(c0, qf[pl * 4 + 2][0], qf[pl * 4 + 2][1], qf[pl * 4 + 2][2], qf[pl * 4 + 2][3], k1[0], k1[1]);
            mma_16816(c1, qf[pl * 4 + 3][0], qf[pl * 4 + 3][1], qf[pl * 4 + 3][2], qf[pl * 4 + 3][3], k1[2], k1[3]);
          } else {
            const uint32_t qa = q_off + (mt * kPl + pl) * 2048;
            uint32_t q0[4], q1[4], q2[4], q3[4];
            ldsm4(q0, qa);
            ldsm4(q1, qa ^ 32);
            ldsm4(q2, qa ^ 64);
            ldsm4(q3, qa ^ 96);
            mma_16816(c0, q0[0], q0[1], q0[2], q0[3], k0[0], k0[1]);
            mma_16816(c1, q1[0], q1[1], q1[2], q1[3], k0[2], k0[3]);
            mma_16816(c0, q2[0], q2[1], q2[2], q2[3], k1[0], k1[1]);
            mma_16816(c1, q3[0], q3[1], q3[2], q3[3], k1[2], k1[3]);
          }
        }
        if (key_head[mt][0] == m) {
          s[mt][0] = c0[0] + c1[0];
          s[mt][1] = c0[1] + c1[1];
        }
        if (key_head[mt][1] == m) {
          s[mt][2] = c0[2] + c1[2];
          s[mt][3] = c0[3] + c1[3];
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) s[mt][e] = fmaf(s[mt][e], qs, -bv[mt][e]);  // masked: minus infinity
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        float mx = fmaxf(s[mt][2 * q], s[mt][2 * q + 1]);
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        if ((lane & 3) == 0) sMax[((mt0 + mt) * 16 + r0 + q * 8) * 8 + cw] = mx;
      }
    }
    compute_bar<kDThreads>();
    if (MW == 2 && n_stages > 1 && warp == 0) {  // everybody is done with the tile before: its stage is free
      const int t_next = t + n_stages - 1;
      if (t_next < t_end) load_tile(t_next, stage == 0 ? n_stages - 1 : stage - 1);
    }
    // ---- weights ----
#pragma unroll
    for (int mt = 0; mt < MTW; ++mt) {
      float al[2];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int row = (mt0 + mt) * 16 + r0 + q * 8;
        const float4 x = *reinterpret_cast<const float4*>(sMax + row * 8), y = *reinterpret_cast<const float4*>(sMax + row * 8 + 4);
        const float mx = fmaxf(fmaxf(fmaxf(x.x, x.y), fmaxf(x.z, x.w)), fmaxf(fmaxf(y.x, y.y), fmaxf(y.z, y.w)));
        const float mn = fmaxf(mrow[mt][q], mx);
        al[q] = mrow[mt][q] == -INFINITY ? 0.f : exp2f(mrow[mt][q] - mn);
        mrow[mt][q] = mn;
        const float base = mn == -INFINITY ? 0.f : mn;
        const float p0 = exp2f(s[mt][2 * q] - base), p1 = exp2f(s[mt][2 * q + 1] - base);
        lrow[mt][q] = lrow[mt][q] * al[q] + p0 + p1;
        *reinterpret_cast<uint32_t*>(sP + (row * kPPitch + cw * 8 + cq) * 2) = pack_bf16x2(p0, p1);
      }
      if (__any_sync(0xffffffffu, al[0] != 1.f || al[1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < NTW; ++i) {
          acc[mt][i][0] *= al[0];
          acc[mt][i][1] *= al[0];
          acc[mt][i][2] *= al[1];
          acc[mt][i][3] *= al[1];
        }
      }
    }
    compute_bar<kDThreads>();
    // ---- products: this warp's heads x its value columns ----
#pragma unroll
    for (int kk = 0; kk < kDT / 16; ++kk) {
      uint32_t pf[MTW][4];
#pragma unroll
      for (int mt = 0; mt < MTW; ++mt) ldsm4(pf[mt], p_off + (mt * 16 * kPPitch + kk * 16) * 2);
#pragma unroll
      for (int i = 0; i < kPairs; ++i) {
        if (nt0 + 2 * i < n_cols) {
          uint32_t vf[4];
          ldsm4_t(vf, kVReg ? kts + v_pair[kVReg ? i : 0] + kk * 2048 : (kts + v_off + kk * 2048 + (i >> 2) * (kDT * 128)) ^ ((i & 3) * 32));
#pragma unroll
          for (int mt = 0; mt < MTW; ++mt) {
            mma_16816(acc[mt][2 * i], pf[mt][0], pf[mt][1], pf[mt][2], pf[mt][3], vf[0], vf[1]);
            mma_16816(acc[mt][2 * i + 1], pf[mt][0], pf[mt][1], pf[mt][2], pf[mt][3], vf[2], vf[3]);
          }
        }
      }
    }
    if (MW == 1) {
      __syncwarp();
      if (lane == 0) mbar_arrive(&empty[stage]);
    } else if (n_stages == 1) {
      compute_bar<kDThreads>();
      if (warp == 0 && t + 1 < t_end) load_tile(t + 1, 0);
    }
    if (++stage == n_stages) {
      stage = 0;
      phase ^= 1;
    }
  }
  compute_bar<kDThreads>();
  // ---- row sums over the warps ----
#pragma unroll
  for (int mt = 0; mt < MTW; ++mt)
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      float l = lrow[mt][q];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      if ((lane & 3) == 0) sMax[((mt0 + mt) * 16 + r0 + q * 8) * 8 + cw] = l;
    }
  compute_bar<kDThreads>();
  float* prod = reinterpret_cast<float*>(sKV);   // [H][G * D]
  const size_t part = ((size_t)b * a.splits + split) * H;
#pragma unroll
  for (int mt = 0; mt < MTW; ++mt)
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int h = (mt0 + mt) * 16 + r0 + q * 8;
      if (h >= H) continue;
      float l = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) l += sMax[h * 8 + w];
      const float inv = a.splits == 1 ? (l > 0.f ? 1.f / l : 0.f) : 1.f;
      float* dst = a.splits == 1 ? prod + (size_t)h * GD : a.part_o + (part + h) * GD;
#pragma unroll
      for (int i = 0; i < NTW; ++i)
        if (nt0 + i < n_cols)
          *reinterpret_cast<float2*>(dst + (nt0 + i) * 8 + cq) = make_float2(acc[mt][i][2 * q] * inv, acc[mt][i][2 * q + 1] * inv);
      if (a.splits > 1 && cw == 0 && (lane & 3) == 0)
        *reinterpret_cast<float2*>(a.part_ml + (part + h) * 2) = make_float2(mrow[mt][q], l);
    }
  if (a.splits > 1) {
    __threadfence();
    compute_bar<kDThreads>();
    if (tid == 0) {
      const int ticket = atomicAdd(a.tickets + b, 1);
      *s_last = ticket == a.splits - 1;
      if (*s_last) a.tickets[b] = 0;
    }
    compute_bar<kDThreads>();
    if (!*s_last) return;
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
    compute_bar<kDThreads>();
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
  compute_bar<kDThreads>();
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
  int mw, mtw, ntw, stages;
  size_t smem;
};
// picks the template and the number of stages; mw = 0: not served
DecPlan plan_decode_kernel(int H, int G, int D) {
  DecPlan d{0, 0, 0, 0, 0};
  if ((D != 64 && D != 128) || H > 64 || H % G != 0) return d;
  const int mw = H <= 16 ? 1 : 2, mtw = H <= 32 ? 1 : 2, mt = mw * mtw;
  const int npw = (G * D / 8 + 7) / 8;
  int ntw = 2;
  while (ntw < npw) ntw *= 2;
  if (ntw > 16 || mtw * ntw > 16) return d;
  const size_t stage = (size_t)kDT * G * D * 2;
  const size_t fixed = (size_t)mt * 16 * D * 2 + (size_t)mt * 16 * kPPitch * 2 + (size_t)mt * 16 * 32 + (size_t)G * D * 2 + (size_t)(H * H + 1) * 4 + 96;
  const size_t prod = (size_t)H * G * D * 4;
  const size_t budget = (size_t)(mw == 1 && ntw <= 4 ? 112 : 224) * 1024;  // two CTAs per SM or one
  int st = 4;
  while (st > 1 && st * stage + fixed > budget) --st;
  if (st * stage < prod || st * stage + fixed > budget) return d;
  d.mw = mw; d.mtw = mtw; d.ntw = ntw; d.stages = st; d.smem = st * stage + fixed;
  return d;
}

template <int D, int MW, int MTW, int NTW>
void launch_decode_t(const TalkDecodeArgs& a, const DecPlan& d, cudaStream_t s) {
  auto kernel = talk_decode_kernel<D, MW, MTW, NTW>;
  AGRPO_SET_MAX_DYN_SMEM(kernel, 226 * 1024, "talk_decode smem attr");
  AGRPO_PREFER_SMEM(kernel);
  const CUtensorMap tk = make_tmap_2d(a.k_cache, D, (uint64_t)a.at.num_cache_blocks * a.at.G * 16, D, 64, 16);
  launch_kernel(kernel, dim3(a.splits, a.at.T), dim3(MW == 1 ? 288 : 512), d.smem, s, "talk_decode", tk, a, d.stages);
}
template <int D, int MW, int MTW>
void launch_decode_n(const TalkDecodeArgs& a, const DecPlan& d, cudaStream_t s) {
  if (d.ntw == 2) return launch_decode_t<D, MW, MTW, 2>(a, d, s);
  if (d.ntw == 4) return launch_decode_t<D, MW, MTW, 4>(a, d, s);
  if (d.ntw == 8) return launch_decode_t<D, MW, MTW, 8>(a, d, s);
  if constexpr (MTW == 1) {
    if (d.ntw == 16) return launch_decode_t<D, MW, MTW, 16>(a, d, s);
  }
  throw std::runtime_error("talk_decode: shape not served");
}
template <int D>
void launch_decode_d(const TalkDecodeArgs& a, const DecPlan& d, cudaStream_t s) {
  if (d.mw == 1) launch_decode_n<D, 1, 1>(a, d, s);
  else if (d.mtw == 1) launch_decode_n<D, 2, 1>(a, d, s);
  else launch_decode_n<D, 2, 2>(a, d, s);
}

}  // namespace

void launch_gather_pages(const void* cache, const int* pages, int n_pages, const int* block_tables, int max_blocks, void* out, int G, int D,
                         int num_cache_blocks, int* status, cudaStream_t s) {
  if (n_pages == 0) return;
  gather_keys_kernel<<<n_pages, 128, 0, s>>>((const bf16*)cache, reinterpret_cast<const int2*>(pages), block_tables, max_blocks, (bf16*)out, G, D,
                                             num_cache_blocks, status);
  check_cuda(cudaGetLastError(), "gather_pages");
}

bool launch_talk_attn_prefill(const WindowAttnArgs& a, const int* tiles, int n_tiles, const int* pages, int n_pages, void* keys, void* acc,
                              cudaStream_t s) {
  if ((a.D != 64 && a.D != 128) || a.block_size != 16 || a.H % a.G != 0) return false;
  const int grp8 = (a.H / a.G + 7) & ~7;
  const size_t mix_smem = (size_t)a.G * a.H * grp8 * 4;
  if (mix_smem > 200 * 1024) return false;
  if (a.T == 0 || n_tiles == 0) return true;
  launch_gather_pages(a.k_cache, pages, n_pages, a.block_tables, a.max_blocks, keys, a.G, a.D, a.num_cache_blocks, a.status, s);
  const int mc_max = 256 / a.D;
  const int chunks = (a.G + mc_max - 1) / mc_max;
  const CUtensorMap tq = make_tmap_2d(a.q, (uint64_t)a.H * a.D, a.T, a.ldq, 64, kPM);
  const CUtensorMap tk = make_tmap_2d(keys, (uint64_t)a.G * a.D, (uint64_t)n_pages * 16, (uint64_t)a.G * a.D, 64, kPN);
  TalkPrefillParams p;
  p.tiles = reinterpret_cast<const int4*>(tiles);
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
  p.status = a.status;
  if (a.D == 128) launch_prefill_t<128>(tq, tk, p, n_tiles, chunks, s);
  else launch_prefill_t<64>(tq, tk, p, n_tiles, chunks, s);
  AGRPO_SET_MAX_DYN_SMEM(talk_mix_gate_kernel, 200 * 1024, "talk_mix smem attr");
  launch_kernel(talk_mix_gate_kernel, dim3((a.T + kMixTokens - 1) / kMixTokens), dim3(kMixThreads), mix_smem, s, "talk_mix_gate",
                (const bf16*)acc, (const bf16*)a.talk, (const bf16*)a.gate, a.ldg, (bf16*)a.out, a.ldo, a.T, a.H, a.G, a.D);
  return true;
}

int talk_decode_ctas_per_sm(int H, int G, int D) {
  const DecPlan d = plan_decode_kernel(H, G, D);
  return d.mw == 0 ? 0 : (d.mw == 1 && d.ntw <= 4 ? 2 : 1);
}

void launch_talk_attn_decode(const TalkDecodeArgs& a, cudaStream_t s) {
  const DecPlan d = plan_decode_kernel(a.at.H, a.at.G, a.at.D);
  if (d.mw == 0 || a.at.block_size != 16 || a.splits < 1 || a.splits > 8) throw std::runtime_error("talk_decode: shape not served");
  if (a.at.T == 0) return;
  if (a.at.D == 128) launch_decode_d<128>(a, d, s);
  else launch_decode_d<64>(a, d, s);
}

}  // namespace agrpo
