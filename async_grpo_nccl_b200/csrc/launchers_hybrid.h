// Launchers of the mechanisms of hybrid attention / scan decoders: zero-centred RMS norms, norm + rotation of whole query / key
// projections, attention inside position chunks, selective scans, and the GEMMs of a parallel block. `fp32` selects 32-bit
// activations and parameters, otherwise both are bf16; the residual stream and recurrent state are always fp32.
#pragma once
#include <cuda_runtime.h>

#include "launchers_layers.h"

namespace agrpo {

// One consumer of the residual stream: h = x * (1 + w) (w nullptr: x itself); h nullptr = absent.
struct NormOut {
  void* h;
  long long ld;
  const void* w;
};

// x[t] = table[ids[t]] * scale (fp32). Fused form of the following norms: out[i] = x * (1 + w_i) without the division by the root
// mean square, whose sums of squares go to ss[t] when out[0] has a weight (30-bit fixed point; ss has n_stats rows of `ss_pitch`, all
// others are cleared):
// the consuming GEMM scales its rows. copy, when given, receives x rounded to the activation type.
struct EmbedArgs {
  const int* ids;
  const void* table;
  float scale;
  float* x;
  void* copy;
  long long ld_copy;
  NormOut out[2];
  long long* ss;
  int n_stats;
  long long ss_pitch;
  int T, W, V;
};
void launch_embed_norm(bool fp32, const EmbedArgs& a, cudaStream_t s);

// out[i][t] = x[t] / sqrt(mean(x[t]^2) + eps) * (1 + w_i); the mean is over `width` channels (padding beyond it is zero).
void launch_rms_rows(bool fp32, const float* x, long long ldx, const NormOut out[2], float eps, int width, int T, int W, cudaStream_t s);
// z = cap * tanh(z / cap)
void launch_softcap_rows(float* z, long long ld, int rows, int V, float cap, cudaStream_t s);

// u [T, ldu] = q | k | v. q and k are divided by the root mean square of their whole projection (H * dim and G * dim values; sums
// from ss_q / ss_k when given), multiplied by plain weights, rotated (dimension i of a head with i + rot / 2, tables [positions,
// rot / 2]) and written in place (q) and to the paged cache (k; v as it is).
struct QkRopeArgs {
  void* u;
  long long ldu;
  const void* q_norm;
  const void* k_norm;
  float eps;
  const long long* ss_q;
  const long long* ss_k;
  const float* cos_t;
  const float* sin_t;
  int max_pos;
  const int* rows;
  const int* seq_lens;
  const int* block_tables;
  int max_blocks;
  void* k_cache;           // [blocks, G, block_size, D]
  void* v_cache;           // [blocks, G, block_size, E]
  int H, G, D, E, dim, rot;
  int block_size, num_cache_blocks, T;
  int* status;
};
void launch_qk_norm_rope(bool fp32, const QkRopeArgs& a, cudaStream_t s);

// Attention of position i over the cached positions j <= i of its own chunk (floor(j / chunk) == floor(i / chunk)):
// softmax of cap * tanh(q.k * scale / cap) (cap 0: no cap).
struct ChunkAttnArgs {
  const void* q;           // [T, ldq], head h at h * D
  long long ldq;
  const void* k_cache;
  const void* v_cache;
  const int* rows;
  const int* seq_lens;
  const int* block_tables;
  int max_blocks;
  float scale, softcap;
  int chunk;
  void* out;               // [T, ldo], head h at h * E
  long long ldo;
  int T, H, G, D, E, block_size, num_cache_blocks;
  int* status;
};
void launch_chunk_attn(bool fp32, const ChunkAttnArgs& a, cudaStream_t s);  // any head sizes up to 512

// Tensor-core form for prompts (bf16, D and E 64 or 128, block_size 16); q points at a matrix of q_cols columns (tensor maps need
// its true extent). Tables as in launch_talk_attn_prefill. False (nothing launched) when the shape is not served.
bool launch_chunk_attn_prefill(const ChunkAttnArgs& a, int q_cols, const int* tiles, int n_tiles, const int* pages, int n_pages, void* keys,
                               void* values, cudaStream_t s);

// Decode step of the mixer after its projection u = q | k | v: norm, rotation, cache write and attention in one kernel (row = slot).
struct ChunkDecodeArgs {
  QkRopeArgs qk;           // rows unused; u is not modified
  ChunkAttnArgs at;        // q unused
  int splits;
  float* part_o;           // [B, H, splits, E]
  float* part_ml;          // [B, H, splits, 2]
  int* tickets;            // [B, H], zero-initialised, re-armed by the kernel
};
bool chunk_decode_serves(int H, int G, int D, int E);
void launch_chunk_attn_decode(const ChunkDecodeArgs& a, cudaStream_t s);

// Pages of a cache [blocks, G, 16, D] as one matrix [16 n_pages, G * D].
void launch_gather_pages(const void* cache, const int* pages, int n_pages, const int* block_tables, int max_blocks, void* out, int G, int D,
                         int num_cache_blocks, int* status, cudaStream_t s);

// Selective scan. xc [T, ldx]: convolved input; r [T, ldr] fp32: step-size code (rank) | B (N) | C (N); z [T, ldz]: gate.
//   dt = softplus(W_dt r_dt + dt_b); S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c xc_c B_n; y_c = sum_n S[c, n] C_n + D_c xc_c
// out = y * silu(z). State [slots, C, N] fp32 (slots state_pitch apart), zero before position 0. Prompts: segs [n, 4] = {first row,
// rows, slot, position of the first row}; decode (segs nullptr): row = slot at position seq_lens - 1.
struct ScanArgs {
  const void* xc;
  long long ldx;
  const float* r;
  long long ldr;
  const void* code;        // packed form: step-size code
  long long ldcode;
  const void* z;
  long long ldz;
  const void* wdt;         // [C, ldw], columns beyond rank are zero
  long long ldw;
  const float* dt_b;       // [C]
  const float* a;          // [C, N]: A
  const float* d;          // [C]
  float* state;
  long long state_pitch;
  const int* segs;
  int n_segs;
  const int* seq_lens;
  void* out;
  long long ldo;
  int T, C, N, rank;
};
void launch_selective_scan_plain(bool fp32, const ScanArgs& a, cudaStream_t s);
// bf16, N up to 64, packed: the step-size code by itself (bf16 rows scan_code_pitch(rank) apart), r = for each quarter of the
// states n values of B, n of C (n = scan_states_per_lane(N)); a in log2 units; a and the state have 4 n entries per channel, zero
// beyond N.
int scan_states_per_lane(int N);   // 0: not served
int scan_code_pitch(int rank);     // rank rounded up to a multiple of 16, and eight more
bool selective_scan_serves(int N, int rank);
bool launch_selective_scan(const ScanArgs& a, cudaStream_t s);   // false (nothing launched): not served

// Both projections of a parallel block in one GEMM: h [M, lda] holds two inputs side by side, `a2` columns apart; the first n1 rows of
// w read the first, the others the second. u = first product, act = relu(second)^2. Rows are scaled by 1 / sqrt(ss_in / width + eps)
// when ss_in is given. Columns [0, q_end) and [q_end, k_end) of u add their squares to ss_q / ss_k (fixed point) when given.
struct ParallelProjArgs {
  const void* h;
  long long lda;
  int a2;
  const void* w;
  long long ldw;
  int M, n1, n2, K;
  void* u;
  long long ldu;
  void* act;
  long long ldact;
  const long long* ss_in;
  int width;
  float eps;
  long long* ss_q;
  long long* ss_k;
  int q_end, k_end;
  int* status;
};
void launch_gemm_parallel_proj(const ParallelProjArgs& a, int num_sms, cudaStream_t s);

// x = (accumulate ? x : 0) + a . w^T (fp32 residual stream), followed by up to two consumers h_i = x * (1 + w_i) and the sums of
// squares of the new rows (ss, fixed point).
struct ResidualArgs {
  const void* a;
  long long lda;
  const void* w;
  long long ldw;
  int M, N, K;
  float* x;
  long long ldx;
  int accumulate;
  NormOut out[2];
  long long* ss;
  int* status;
};
void launch_gemm_residual(const ResidualArgs& a, int num_sms, cudaStream_t s);

// Product whose first n1 columns are stored as bf16 and the others as fp32 (both multiples of 8).
struct SplitStoreArgs {
  const void* a;
  long long lda;
  const void* w;
  long long ldw;
  int M, n1, n2, K;
  void* d16;
  long long ld16;
  float* d32;
  long long ld32;
  int* status;
};
void launch_gemm_split_store(const SplitStoreArgs& a, int num_sms, cudaStream_t s);

}  // namespace agrpo
