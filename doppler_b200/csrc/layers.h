// Launchers of the kernels a decoder described layer by layer is built from (stack.cu schedules them).
#pragma once
#include "common.h"

// Which sequence and position a row of a launch belongs to: decode rows are sequences 0..rows-1 at pos[row];
// a portion's rows are consecutive positions of one sequence from start_pos on.
struct RowMap {
  const int *pos = nullptr;  // device, decode
  int start_pos = 0, seq = 0;
};

// ---- residual streams, grouped RMSNorm, input convolution (streams.cu) ----
constexpr int DP_MAX_STREAMS = 16;

// What a sublayer does on entry to the rows it reads: u = sum_s in[s] x_s, grouped RMSNorm, h + causal conv of h.
struct SublayerIn {
  const float *in = nullptr;              // [streams]
  const __nv_bfloat16 *norm_w = nullptr;  // [width]
  const __nv_bfloat16 *conv_w = nullptr;  // [width, taps], taps > 0
  int taps = 0, groups = 1;
  float eps = 0.0f;
  // history of h: position p of sequence q lives in hist + q * hist_seq + (p % taps) * width
  float *hist = nullptr;
  size_t hist_seq = 0;
  float *stage = nullptr;                 // same layout, one sequence: where a portion leaves its last rows (see dpk_hist_commit)
};
// The end of a sublayer: x_t <- sum_s mix[s][t] x_s + out[t] y, with y through a grouped RMSNorm first where norm_w is set
struct SublayerOut {
  const float *mix = nullptr, *out = nullptr;  // [streams, streams] (from, to), [streams]
  const __nv_bfloat16 *norm_w = nullptr;       // [width]
  int groups = 1;
  float eps = 0.0f;
};

// One sublayer boundary over `rows` rows of x [rows][streams][width]: write y of the sublayer that ended into the
// streams (y null: x is already current and x_out is not written), then prepare the input of the next sublayer,
// dst [rows][dst_stride], bf16 or f32.  x_out must not alias x.
dp_status dpk_stream_boundary(dp_ctx *ctx, const float *x, float *x_out, const float *y, const SublayerOut &end, const SublayerIn &next,
                              int streams, int width, void *dst, bool dst_bf16, int dst_stride, int rows, const RowMap &map);
// the end of the last layer: h[row] = sum of the streams after y has been written into them
dp_status dpk_stream_sum(dp_ctx *ctx, const float *x, const float *y, const SublayerOut &end, int streams, int width, float *h, int rows);
// x[row][s] = table[ids[row]] * scale for every stream; u (optional) [row] = (sum_s in[s]) * x
dp_status dpk_stream_embed(dp_ctx *ctx, const int *ids, const __nv_bfloat16 *table, int table_stride, float scale, int streams, int width, float *x,
                           const float *in, float *u, int rows);
// rows of `width` values: RMSNorm of every one of `groups` parts, times w; dst bf16 or f32.  w_shared: one weight of a
// part's size serves all parts.  gate (optional, rows of gate_stride floats): the result times sigmoid(gate).
struct GroupNorm {
  const __nv_bfloat16 *w = nullptr;
  int groups = 1;
  float eps = 0.0f;
  bool w_shared = false;
  const float *gate = nullptr;
  int gate_stride = 0;
};
dp_status dpk_group_norm(dp_ctx *ctx, const float *x, int x_stride, const GroupNorm &n, int width, void *dst, bool dst_bf16, int dst_stride, int rows);
// copies the staged last rows of a portion into the histories of sequence `seq`: entries of {stage, hist, hist_seq, channels, taps}
struct HistEntry {
  const float *stage;
  float *hist;
  unsigned long long hist_seq;
  int channels, taps;
};
dp_status dpk_hist_commit(dp_ctx *ctx, const HistEntry *entries, int n_entries, int max_channels, int rows, int start_pos, int seq);

// ---- bf16 weights ----
// One-row products (gemv_bf16.cu): y = W x with x built by the kernel's prologue in f32 and the result handed to an
// epilogue.  W bf16 [N, K], rows of w_stride elements (multiple of 8, zero padded).
enum { GEMV_SRC_PLAIN = 0, GEMV_SRC_NORM = 1, GEMV_SRC_ATTN = 2, GEMV_SRC_RESIDUAL = 3, GEMV_SRC_GATED = 4 };
enum { GEMV_DST_PLAIN = 0, GEMV_DST_GLU = 1, GEMV_DST_STREAMS = 2 };
struct GemvBf16 {
  const __nv_bfloat16 *w = nullptr;
  int N = 0, K = 0, w_stride = 0;
  const float *x = nullptr;   // PLAIN: the vector; NORM: the row to normalise; ATTN: split partials [head][split][vdim + 2]
  SublayerIn norm;            // NORM (in / stage unused)
  const int *pos = nullptr;   // NORM with an input convolution: position of the token
  // RESIDUAL: the row to normalise is x + res.out[0] * norm(res_y) (one stream), which is also stored to x_out
  SublayerOut res;
  const float *res_y = nullptr;
  float *x_out = nullptr;
  // GATED: the norm's weight serves every group; its result times sigmoid(gate), one gate per value
  bool norm_w_shared = false;
  // ATTN
  const float *gate = nullptr;  // per head, null: none (GATED: per value)
  int heads = 0, vdim = 0, splits = 0;
  float *y = nullptr;         // PLAIN, GLU: the output vector
  // GLU: rows come in groups of sixteen, eight gate rows and their eight up rows; N / 2 outputs
  float limit = 0.0f, slope = 1.0f, shift = 0.0f;
  // STREAMS: the streams (in place), the sublayer's vectors, and u of the next sublayer (next_in null: all ones)
  SublayerOut end;
  int streams = 1;
  float *streams_x = nullptr;
  const float *next_in = nullptr;
  float *next_u = nullptr;
  uint32_t prefetch_bytes = 4096;  // per row, before the previous kernel has finished
};
dp_status dpk_gemv_bf16(dp_ctx *ctx, int src, int dst, const GemvBf16 &p);

// Products of several rows: C [M, N] f32 = A [M, K] W^T.  glu: rows of W in groups of sixteen as above, the activation
// [M, N / 2] is stored to glu_dst in A's type instead (rows of glu_stride elements).
struct GluOut {
  void *dst = nullptr;
  int stride = 0;
  float limit = 0.0f, slope = 1.0f, shift = 0.0f;
};
// decay: C is exp(-rate[n] softplus(c + bias[n])) instead (c: the product)
struct DecayOut {
  const float *rate = nullptr, *bias = nullptr;  // [N]
};
dp_status dpk_gemm_bf16_tc(dp_ctx *ctx, const __nv_bfloat16 *W, int w_stride, const __nv_bfloat16 *A, int a_stride, float *C, int M, int N, int K,
                           const GluOut *glu, const DecayOut *decay = nullptr);
dp_status dpk_gemm_bf16w_f32(dp_ctx *ctx, const __nv_bfloat16 *W, int w_stride, const float *A, int a_stride, float *C, int M, int N, int K,
                             const GluOut *glu, const DecayOut *decay = nullptr);
// f16 operands, f16 result: C [M, N] = A [M, K] W^T (f32 accumulation)
dp_status dpk_gemm_f16_tc(dp_ctx *ctx, const __half *W, int w_stride, const __half *A, int a_stride, __half *C, int c_stride, int M, int N, int K);

// ---- attention helpers (attn_prep.cu) ----
// rows [q | k | v | ...] of qkv_stride floats: q and k per head optionally divided by their root mean square; q to
// q_out [row][heads][dim] f32, k and v appended to the caches (f16 or f32) at their positions
dp_status dpk_unit_qk_kv(dp_ctx *ctx, const float *qkv, int qkv_stride, float *q_out, void *kc, void *vc, bool kv_f32, int heads, int kv_heads, int dim,
                         int vdim, bool unit_rms, float eps, size_t k_seq, size_t v_seq, int rows, const RowMap &map);

// ---- Mamba-2 (ssm.cu) ----
// Linear attention with one constant decay per head is the same recurrence: x = v, B = k, C = q, every head a group of its
// own, step size 1 (SsmWeights::decay set, dt_bias null), no convolution (taps 1, conv null), no skip (d null), and the
// gate, in z's place, left to what follows (gated false).
struct SsmShape {
  int heads, vdim, state, groups, taps;
  int state_stride;  // padded state size: 32 * a power of two
  bool gated = true; // the output times silu(z)
};
int dpk_ssm_state_stride(int state);  // 0: too large
struct SsmWeights {
  const float *conv = nullptr, *conv_b = nullptr, *dt_bias = nullptr;  // conv [channels, taps]
  const float *a = nullptr;      // [heads] decay exponent per unit step: -exp(A_log), or the logarithm of decay
  const float *d = nullptr;
  const float *decay = nullptr;  // [heads] constant decay (step size 1)
};
// conv histories as in SublayerIn; S: state of sequence q at s + q * s_seq, [head][vdim][state_stride]
struct SsmState {
  float *hist = nullptr;
  size_t hist_seq = 0;
  float *stage = nullptr;
  float *s = nullptr;
  size_t s_seq = 0;
};
// One token per row, rows are sequences: convolution, step size, state update and output of every head, times silu(z).
// proj [row][z | x | B | C | dt] of proj_stride floats -> out [row][heads * vdim]
dp_status dpk_ssm_step(dp_ctx *ctx, const float *proj, int proj_stride, const SsmShape &sh, const SsmWeights &w, const SsmState &st, float *out, int rows,
                       const int *pos);
// Consecutive tokens of one sequence: the convolution (xbc [rows][channels], f32 or bf16) and step sizes (dt [rows][heads]),
// then the recurrence, token by token in f32 (dpk_ssm_scan, any shape) or in chunks on the tensor cores with bf16 x, B
// and C (dpk_ssm_chunk)
dp_status dpk_ssm_conv(dp_ctx *ctx, const float *proj, int proj_stride, const SsmShape &sh, const SsmWeights &w, const SsmState &st, void *xbc, bool bf16,
                       float *dt, int rows, const RowMap &map);
bool dpk_ssm_chunk_ok(const SsmShape &sh, int rows);
dp_status dpk_ssm_chunk(dp_ctx *ctx, const float *proj, int proj_stride, const __nv_bfloat16 *xbc, const float *dt, const SsmShape &sh, const SsmWeights &w,
                        const SsmState &st, float *out, int rows, const RowMap &map);
dp_status dpk_ssm_scan(dp_ctx *ctx, const float *proj, int proj_stride, const float *xbc, const float *dt, const SsmShape &sh, const SsmWeights &w,
                       const SsmState &st, float *out, int rows, const RowMap &map);

// ---- gated delta rule with a decay per key channel (delta.cu) ----
struct DeltaShape {
  int heads, kv_heads, dim, vdim, taps, decay_rank, gate_rank;
  int state_stride;  // padded key size: 32 * a power of two (dpk_ssm_state_stride)
  __host__ __device__ int qk() const { return kv_heads * dim; }
  __host__ __device__ int inner() const { return heads * vdim; }
  __host__ __device__ int channels() const { return 2 * qk() + inner(); }       // of the short convolutions: q | k | v
  __host__ __device__ int beta_col() const { return channels(); }                // projection columns behind them
  __host__ __device__ int a1_col() const { return beta_col() + heads; }
  __host__ __device__ int g1_col() const { return a1_col() + decay_rank; }
  __host__ __device__ int proj_cols() const { return g1_col() + gate_rank; }
};
struct DeltaWeights {
  const float *conv = nullptr;                  // [channels, taps]
  const float *rate = nullptr, *bias = nullptr; // [heads * dim]: exp(A_log) of the head, dt_bias
  const __nv_bfloat16 *a2 = nullptr, *g2 = nullptr;
  int a2_stride = 0, g2_stride = 0;
};
// what a portion's tokens bring to the recurrence, f32
struct DeltaRows {
  float *q, *k;     // [rows][kv_heads * dim] unit vectors, q also / sqrt(dim)
  float *v;         // [rows][heads * vdim]
  float *beta;      // [rows][heads]
  const float *g;   // [rows][heads * dim] decays
  float *records;   // dpk_delta_record_floats: the same, arranged for the recurrence
  __nv_bfloat16 *a_low = nullptr, *g_low = nullptr;  // low-rank rows as bf16, strides multiples of 8 (null: not wanted)
  int a_low_stride = 0, g_low_stride = 0;
};
// one token per row, rows are sequences; proj [row][q | k | v | b | a1 | g1]: everything of the mixer between the projection
// and the output norm.  out [row][heads * vdim], gate [row][heads * vdim]: the output gate before its sigmoid
dp_status dpk_delta_step(dp_ctx *ctx, const float *proj, int proj_stride, const DeltaShape &sh, const DeltaWeights &w, const SsmState &st, float *out,
                         float *gate, int rows, const int *pos);
// consecutive tokens of one sequence: convolutions, unit norms, write strengths; then the recurrence over them
dp_status dpk_delta_rows(dp_ctx *ctx, const float *proj, int proj_stride, const DeltaShape &sh, const DeltaWeights &w, const SsmState &st, const DeltaRows &r,
                         int rows, const RowMap &map);
size_t dpk_delta_record_floats(const DeltaShape &sh, int rows);
dp_status dpk_delta_scan(dp_ctx *ctx, const DeltaShape &sh, const SsmState &st, const DeltaRows &r, float *out, int rows, const RowMap &map);

// ---- latent attention (latent.cu) ----
// A cache row is [c (kv_rank) | zeros | rotated key part (rot_dim) | zeros], both parts padded to sixteen values; queries
// brought into the latent space ("absorbed": q' = W_uk^T q) have the same layout, one row per head.
struct LatentShape {
  int heads, dim, vdim, q_rank, kv_rank, rot_dim;
  float eps, scale;
  __host__ __device__ int c_pad() const { return (kv_rank + 15) / 16 * 16; }
  __host__ __device__ int cols() const { return c_pad() + (rot_dim + 15) / 16 * 16; }
  __host__ __device__ int dkv_col() const { return q_rank; }                      // projection columns: dq | dkv | g
  __host__ __device__ int gate_col() const { return q_rank + kv_rank + rot_dim; }
  __host__ __device__ int proj_cols() const { return gate_col() + heads; }
};
struct LatentCache {
  void *rows = nullptr;   // f16, or f32 in the 32-bit mode
  bool f32 = false;
  size_t seq = 0;         // elements between two sequences
};
// cos, sin [position][rot_dim / 2]
struct Rotation {
  const float *cos_t = nullptr, *sin_t = nullptr;
};
// rows of projections: normed latent and rotated key part to the cache; the rotated part of the queries q [row][head][dim + rot_dim]
// in place (q_rot null) or to the tail of q_rot [row][head][cols]
dp_status dpk_latent_append(dp_ctx *ctx, const float *proj, int proj_stride, const LatentShape &sh, const __nv_bfloat16 *norm_w, const Rotation &rot,
                            const LatentCache &cache, float *q, float *q_rot, int rows, const RowMap &map);
// one decode row: the same, and the absorbed queries in one launch (wuk [heads * dim, kv_rank])
dp_status dpk_latent_absorb_step(dp_ctx *ctx, const float *proj, const LatentShape &sh, const __nv_bfloat16 *norm_w, const Rotation &rot, const LatentCache &cache,
                                 const __nv_bfloat16 *wuk, int wuk_stride, const float *q, float *q_abs, const int *pos);
// y[row][z][n] = sum_k x[row][z][k] W[z][n][k] in f32 for every z (head); W element (z, n, k) at W[z * w_z + n * w_n + k * w_k];
// gate (optional) [row][z]: times its sigmoid.  y f32 or bf16, rows of y_row, heads y_z apart.
struct GroupedProduct {
  const __nv_bfloat16 *w = nullptr;
  size_t w_z = 0, w_n = 0, w_k = 0;
  const float *x = nullptr;
  size_t x_row = 0, x_z = 0;
  void *y = nullptr;
  bool y_bf16 = false;
  size_t y_row = 0, y_z = 0;
  const float *gate = nullptr;
  int gate_stride = 0;
  int rows = 0, heads = 0, N = 0, K = 0;
};
dp_status dpk_grouped_product(dp_ctx *ctx, const GroupedProduct &p);
// one row: split partials of the attention in latent space [head][split][c_pad + 2] (splits 1: the merged rows) -> values
// out [head][vdim] = W_uv (merged context), times sigmoid(gate[head])
dp_status dpk_latent_values_step(dp_ctx *ctx, const float *part, int splits, const LatentShape &sh, const __nv_bfloat16 *wuv, int wuv_stride, const float *gate,
                                 float *out);
