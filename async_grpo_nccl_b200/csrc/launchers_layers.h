// Launchers of the listed-layer kernels (Dynamic Tanh norms, short convolutions, windowed attention with mixed heads).
// `fp32` selects 32-bit activations and parameters, otherwise both are bf16; the residual stream is always fp32.
#pragma once
#include <cuda_runtime.h>

namespace agrpo {

struct DytArgs {  // tanh(alpha x) * w + b
  const void* w;
  const void* b;
  const void* alpha;
};

// Tail of a sublayer, fused into the GEMM that produces its output: x += n1(output) (fp32 residual), h = n2(x).
struct DytTail {
  float* x;
  long long ldx;
  void* h;
  long long ldh;
  DytArgs n1, n2;
};

// x[t] = table[ids[t]] * scale (fp32), h[t] = norm(x[t])
void launch_embed_dyt(bool fp32, const int* ids, const void* table, float scale, float* x, void* h, const DytArgs& norm, int T, int W, int V,
                      cudaStream_t s);

// Causal short convolution of the first `q_cols + k_cols` columns of u [T, ldu] (weights [taps, q_cols + k_cols], the current token's last). The q
// part goes to q_out [T, q_cols], the k part to its place in the paged cache [blocks, G, block_size, D]. Values of tokens
// before the segment come from the sequence's ring [slots, ring_len, q_cols + k_cols] (position p at p % ring_len; slots are
// ring_pitch elements apart).
struct ShortConvArgs {
  const void* u;
  long long ldu;
  const void* w;
  int taps;
  void* ring;
  int ring_len;
  long long ring_pitch;
  const int* rows;       // [T, 4], nullptr: decode rows
  const int* seq_lens;
  const int* block_tables;
  int max_blocks;
  void* q_out;
  void* k_cache;
  int q_cols, k_cols, D, block_size, num_cache_blocks, T;
  int* status;
  const void* bias = nullptr;  // [q_cols + k_cols], optional
  int silu = 0;                // 1: y / (1 + e^-y) of the result
};
void launch_short_conv(bool fp32, const ShortConvArgs& a, cudaStream_t s);
// Decode rows only: convolution and ring in one launch.
void launch_short_conv_decode(bool fp32, const ShortConvArgs& a, cudaStream_t s);
// Writes the values that later steps need into the ring: ring_rows lists the last ring_len rows of each segment
// (nullptr: decode rows, every row). A launch of its own: the convolution of a segment's first rows reads the ring.
void launch_short_conv_ring(bool fp32, const ShortConvArgs& a, const int* ring_rows, int n_ring_rows, cudaStream_t s);

// Sliding-window attention over the paged keys (which are also the values), softmax weights mixed across heads by
// talk [H, H], output multiplied by sigmoid(gate). Any head size that is a multiple of 8.
struct WindowAttnArgs {
  const void* q;           // [T, ldq] head h at h * D
  long long ldq;
  const void* k_cache;
  const int* rows;
  const int* seq_lens;
  const int* block_tables;
  int max_blocks;
  const float* bias;       // [H, bias_len], log2 units, subtracted: entry d for distance d
  int bias_len;
  const float* qscale;     // [max positions] score factor of a query at each position, log2 units
  int qscale_len;
  const void* talk;        // [H, H] or nullptr (no mixing)
  const void* gate;        // [T, ldg] pre-activation, or nullptr (no gate)
  long long ldg;
  int window;
  void* out;               // [T, ldo]
  long long ldo;
  int T, H, G, D, block_size, num_cache_blocks;
  int* status;
};
void launch_window_attn(bool fp32, const WindowAttnArgs& a, cudaStream_t s);

// Tensor-core forms (bf16, D = 64 or 128, block_size 16). pages [n_pages, 2] = {slot, page of the sequence}: what the step can see,
// gathered into keys [16 n_pages, G * D]; tiles [n_tiles, 4] = {first row, rows, position of the first row, row of position 0 in
// keys}; acc: scratch [T, H, G, D] bf16. Returns false, having launched nothing, for shapes that are not served.
bool launch_talk_attn_prefill(const WindowAttnArgs& a, const int* tiles, int n_tiles, const int* pages, int n_pages, void* keys, void* acc,
                              cudaStream_t s);
// Decode: short convolution of the new token, attention, mixing, gate and ring / cache update in one kernel (row = slot).
struct TalkDecodeArgs {
  WindowAttnArgs at;      // q unused: the kernel convolves q itself
  const void* u;          // [B, ldu]: q | k | gate
  long long ldu;
  const void* conv_w;
  int taps;
  void* ring;
  int ring_len;
  long long ring_pitch;
  void* k_cache;
  int splits;
  float* part_o;          // [B, splits, H, G, D]
  float* part_ml;         // [B, splits, H, 2]
  int* tickets;           // [B], zero-initialised, re-armed by the kernel
};
int talk_decode_ctas_per_sm(int H, int G, int D);  // 0: shape not served
void launch_talk_attn_decode(const TalkDecodeArgs& a, cudaStream_t s);

// y = a . b^T in true fp32 (no tensor cores), every output summed over K in the same order whatever the batch.
struct GemmF32Post {       // what happens to a result on its way out, in this order
  int relu2 = 0;           // max(y, 0)^2
  float softcap = 0.f;     // > 0: cap * tanh(y / cap)
  int accumulate = 0;      // d += y
};
void launch_gemm_f32(const float* a, long long lda, const float* b, long long ldb, float* d, long long ldd, int M, int N, int K,
                     cudaStream_t s, const GemmF32Post& post = GemmF32Post());
// d = silu(a . bg^T) * (a . bu^T), b = [bg; bu] with 2F rows
void launch_gemm_swiglu_f32(const float* a, long long lda, const float* b, long long ldb, float* d, long long ldd, int M, int F, int K,
                            cudaStream_t s);
// Sublayer tail in the GEMM's epilogue: x += norm1(a . b^T) (fp32 residual), h = norm2(x).
void launch_gemm_dyt_f32(const float* a, long long lda, const float* b, long long ldb, int M, int N, int K, float* x, long long ldx,
                         float* h, long long ldh, const DytArgs& n1, const DytArgs& n2, cudaStream_t s);
void launch_gemm_dyt_bf16(const void* a, long long lda, const void* b, long long ldb, int M, int N, int K, float* x, long long ldx, void* h,
                          long long ldh, const DytArgs& n1, const DytArgs& n2, int* status, int num_sms, cudaStream_t s);

// Sampling from fp32 logits [rows, V]: the same noise stream as the fused lm_head sampler.
void launch_sample_logits(const float* logits, long long ld, int rows, int V, float temperature, const unsigned long long* seeds,
                          int* tokens, float* logprobs, cudaStream_t s);

}  // namespace agrpo
