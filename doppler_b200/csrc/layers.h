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
// The end of a sublayer: x_t <- sum_s mix[s][t] x_s + out[t] y
struct SublayerOut {
  const float *mix = nullptr, *out = nullptr;  // [streams, streams] (from, to), [streams]
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
// rows of `width` values: RMSNorm of every one of `groups` parts, times w; dst bf16 or f32
dp_status dpk_group_norm(dp_ctx *ctx, const float *x, int x_stride, const __nv_bfloat16 *w, int groups, float eps, int width, void *dst, bool dst_bf16,
                         int dst_stride, int rows);
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
enum { GEMV_SRC_PLAIN = 0, GEMV_SRC_NORM = 1, GEMV_SRC_ATTN = 2 };
enum { GEMV_DST_PLAIN = 0, GEMV_DST_GLU = 1, GEMV_DST_STREAMS = 2 };
struct GemvBf16 {
  const __nv_bfloat16 *w = nullptr;
  int N = 0, K = 0, w_stride = 0;
  const float *x = nullptr;   // PLAIN: the vector; NORM: the row to normalise; ATTN: split partials [head][split][vdim + 2]
  SublayerIn norm;            // NORM (in / stage unused)
  const int *pos = nullptr;   // NORM with an input convolution: position of the token
  // ATTN
  const float *gate = nullptr;  // per head, null: none
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
dp_status dpk_gemm_bf16_tc(dp_ctx *ctx, const __nv_bfloat16 *W, int w_stride, const __nv_bfloat16 *A, int a_stride, float *C, int M, int N, int K,
                           const GluOut *glu);
dp_status dpk_gemm_bf16w_f32(dp_ctx *ctx, const __nv_bfloat16 *W, int w_stride, const float *A, int a_stride, float *C, int M, int N, int K,
                             const GluOut *glu);

// ---- attention helpers (attn_prep.cu) ----
// rows [q | k | v | ...] of qkv_stride floats: q and k per head optionally divided by their root mean square; q to
// q_out [row][heads][dim] f32, k and v appended to the caches (f16 or f32) at their positions
dp_status dpk_unit_qk_kv(dp_ctx *ctx, const float *qkv, int qkv_stride, float *q_out, void *kc, void *vc, bool kv_f32, int heads, int kv_heads, int dim,
                         int vdim, bool unit_rms, float eps, size_t k_seq, size_t v_seq, int rows, const RowMap &map);

// ---- Mamba-2 (ssm.cu) ----
struct SsmShape {
  int heads, vdim, state, groups, taps;
  int state_stride;  // padded state size: 32 * a power of two
};
int dpk_ssm_state_stride(int state);  // 0: too large
struct SsmWeights {
  const float *conv, *conv_b, *dt_bias, *a_log, *d;  // conv [channels, taps]
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
