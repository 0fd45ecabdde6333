// Decoders described layer by layer: weights, per-sequence state and the schedule of their layers.
//
// A dp_model whose `stack` is set is run by the same runner as the dense Q4_K decoder (model.cu: portions, decode
// graph, greedy pick, sequence lengths); this file supplies what differs.  Two schedules:
//
//   one decode row     every kernel rebuilds its own input (gemv_bf16.cu), three kernels for a Mamba-2 sublayer
//                      (projection [norm + input convolution] -> step -> output projection [group norm; streams]),
//                      three for an attention sublayer, two for the feed-forward
//   several rows       (portions of a prompt, batched decode) one boundary kernel between two sublayers
//                      (streams.cu), tensor-core products, and the mixers' own kernels
//
// State of a sequence: K/V rows of the attention layers (contiguous, position p at row p), the recurrent state of
// the Mamba-2 layers, and short histories (rings of `taps` positions) of every causal convolution.  None of it is
// read at or beyond the sequence's length, and position 0 starts from zeros, so a slot is reused by setting its
// length to 0.  A portion leaves the last rows of its histories in a stage; one kernel at its end moves them into the
// rings (writing them earlier would overwrite rows other CTAs of the portion still read).
#include "layers.h"
#include "model.h"

#include <cstring>

dp_status dpk_attention_split_only(dp_ctx *ctx, const dpk_attn_params &p, float *scratch, int splits);

namespace {

size_t up(size_t v, size_t a) { return dp_cdiv(v, a) * a; }

struct Mat {
  dp_buf buf = nullptr;
  int N = 0, K = 0, stride = 0;
  const __nv_bfloat16 *w() const { return (const __nv_bfloat16 *)buf->dptr; }
};

struct StackLayer {
  dp_layer_cfg c;
  Mat proj, o, gateup, down;  // proj: q | k | v | head gates, or the Mamba-2 input projection
  __nv_bfloat16 *norm[2] = {}, *conv[2] = {}, *ssm_norm = nullptr;
  float *hc_in[2] = {}, *hc_out[2] = {}, *hc_mix[2] = {};
  float *ssm_conv = nullptr, *ssm_conv_b = nullptr, *dt_bias = nullptr, *a_log = nullptr, *d = nullptr;
  float *hist[2] = {}, *stage[2] = {};
  SsmShape ssm = {};
  SsmState st;
  uint64_t missing = 0;  // bit per dp_tensor_id still to be loaded
  bool attention() const { return c.mixer == DP_MIXER_ATTENTION; }
  int q_cols() const { return c.heads * c.dim; }
  int k_cols() const { return c.kv_heads * c.dim; }
  int v_cols() const { return c.kv_heads * c.vdim; }
  int inner() const { return c.heads * c.vdim; }
  int channels() const { return inner() + 2 * c.groups * c.state; }
  int ff_rows() const { return (int)up((size_t)c.ff, 8); }
};

}  // namespace

struct dp_stack {
  dp_stack_cfg cfg;
  bool f32 = false;
  std::vector<StackLayer> layers;
  Mat embed;
  __nv_bfloat16 *final_norm = nullptr;
  uint64_t missing = 0;
  dp_buf vectors = nullptr, state = nullptr, acts = nullptr, entries = nullptr;
  int n_entries = 0, max_channels = 0;
  size_t state_bytes = 0;
  float *x[2], *y, *proj, *q, *xbc, *dt, *mix, *act_f32;
  void *a, *act;  // inputs of the products (bf16, or f32 in the 32-bit mode)
};

namespace {

dp_status mat_alloc(dp_model *m, Mat *t, int N, int K, const char *label) {
  t->N = N; t->K = K; t->stride = (int)up((size_t)K, 8);
  DP_TRY(dp_buf_acquire(m->ctx, (size_t)N * t->stride * 2, label, &t->buf));
  m->weight_bytes += (size_t)N * t->stride * 2;
  return dp_buf_fill(m->ctx, t->buf, 0, 0, t->buf->bytes);
}

// rows of a host matrix into rows row0.. of a padded one
dp_status mat_upload(dp_ctx *ctx, const Mat &t, int row0, const void *host, int rows, int cols) {
  DP_CUDA(ctx, cudaMemcpy2DAsync((char *)t.buf->dptr + (size_t)row0 * t.stride * 2, (size_t)t.stride * 2, host, (size_t)cols * 2, (size_t)cols * 2, (size_t)rows,
                                 cudaMemcpyHostToDevice, ctx->stream));
  DP_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  return DP_OK;
}

// gate or up rows into their places of the interleaved matrix (groups of eight)
dp_status mat_upload_glu(dp_ctx *ctx, const Mat &t, bool is_up, const void *host, int rows, int cols) {
  const int padded = t.N / 2;
  std::vector<uint16_t> stage((size_t)padded * t.stride, 0);
  for (int r = 0; r < rows; r++) memcpy(stage.data() + (size_t)r * t.stride, (const uint16_t *)host + (size_t)r * cols, (size_t)cols * 2);
  const size_t group = (size_t)8 * t.stride * 2;
  DP_CUDA(ctx, cudaMemcpy2DAsync((char *)t.buf->dptr + (is_up ? group : 0), 2 * group, stage.data(), group, group, (size_t)padded / 8, cudaMemcpyHostToDevice,
                                 ctx->stream));
  DP_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  return DP_OK;
}

dp_status upload_raw(dp_ctx *ctx, void *dst, const void *src, size_t bytes) {
  DP_CUDA(ctx, cudaMemcpyAsync(dst, src, bytes, cudaMemcpyHostToDevice, ctx->stream));
  DP_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  return DP_OK;
}

dp_status upload_as_f32(dp_ctx *ctx, float *dst, const void *host_bf16, size_t n) {
  std::vector<float> v(n);
  for (size_t i = 0; i < n; i++) {
    const uint32_t bits = (uint32_t)((const uint16_t *)host_bf16)[i] << 16;
    memcpy(&v[i], &bits, 4);
  }
  return upload_raw(ctx, dst, v.data(), n * 4);
}

// carves typed pieces out of one allocation: a first pass adds up sizes, a second hands out addresses
struct Carver {
  char *base = nullptr;
  size_t off = 0;
  template <typename T> void take(T **p, size_t n) {
    if (base) *p = reinterpret_cast<T *>(base + off);
    off += up(n * sizeof(T), 256);
  }
};

void carve_vectors(dp_stack *s, Carver &c) {
  const size_t H = s->cfg.width, S = s->cfg.streams, taps = s->cfg.input_taps;
  c.take(&s->final_norm, H);
  for (StackLayer &L : s->layers) {
    for (int q = 0; q < (L.c.ff ? 2 : 1); q++) {
      c.take(&L.norm[q], H);
      if (taps) c.take(&L.conv[q], H * taps);
      c.take(&L.hc_in[q], S); c.take(&L.hc_out[q], S); c.take(&L.hc_mix[q], S * S);
    }
    if (!L.attention()) {
      c.take(&L.ssm_conv, (size_t)L.channels() * L.c.conv_taps); c.take(&L.ssm_conv_b, L.channels());
      c.take(&L.dt_bias, L.c.heads); c.take(&L.a_log, L.c.heads); c.take(&L.d, L.c.heads);
      c.take(&L.ssm_norm, L.inner());
    }
  }
}

void carve_state(dp_stack *s, Carver &c) {
  const size_t H = s->cfg.width, B = s->cfg.max_batch, taps = s->cfg.input_taps;
  for (StackLayer &L : s->layers) {
    if (taps > 1)
      for (int q = 0; q < (L.c.ff ? 2 : 1); q++) { c.take(&L.hist[q], B * taps * H); c.take(&L.stage[q], taps * H); }
    if (!L.attention()) {
      L.st.hist_seq = (size_t)L.c.conv_taps * L.channels();
      L.st.s_seq = (size_t)L.inner() * L.ssm.state_stride;
      c.take(&L.st.hist, B * L.st.hist_seq); c.take(&L.st.stage, L.st.hist_seq); c.take(&L.st.s, B * L.st.s_seq);
    }
  }
}

void carve_acts(dp_model *m, Carver &c) {
  dp_stack *s = m->stack;
  const size_t T = m->T, H = s->cfg.width, S = s->cfg.streams;
  size_t proj = 0, q = 1, xbc = 1, heads = 1, mix = 1, k = up(H, 8), ff = 1;
  for (const StackLayer &L : s->layers) {
    if ((size_t)L.proj.N > proj) proj = L.proj.N;
    if ((size_t)L.o.stride > k) k = L.o.stride;
    if ((size_t)L.inner() > mix) mix = L.inner();
    if (L.c.ff && (size_t)L.ff_rows() > ff) ff = L.ff_rows();
    if (L.attention()) { if ((size_t)L.q_cols() > q) q = L.q_cols(); }
    else {
      if ((size_t)L.channels() > xbc) xbc = L.channels();
      if ((size_t)L.c.heads > heads) heads = L.c.heads;
    }
  }
  c.take(&s->x[0], T * S * H); c.take(&s->x[1], T * S * H); c.take(&s->y, T * H); c.take(&m->h, T * H);
  c.take(&s->proj, T * proj); c.take(&s->q, T * q); c.take(&s->xbc, T * xbc); c.take(&s->dt, T * heads); c.take(&s->mix, T * mix);
  const size_t e = s->f32 ? 4 : 2;
  char *a = nullptr, *act = nullptr;
  c.take(&a, T * k * e); c.take(&act, T * ff * e); c.take(&s->act_f32, ff);
  s->a = a; s->act = act;
}

SublayerIn sub_in(const dp_stack *s, const StackLayer &L, int q) {
  SublayerIn n;
  n.in = L.hc_in[q]; n.norm_w = L.norm[q]; n.conv_w = L.conv[q];
  n.taps = s->cfg.input_taps; n.groups = s->cfg.norm_groups; n.eps = s->cfg.eps;
  n.hist = L.hist[q]; n.hist_seq = (size_t)s->cfg.input_taps * s->cfg.width; n.stage = L.stage[q];
  return n;
}

SublayerOut sub_out(const StackLayer &L, int q) {
  SublayerOut o;
  o.mix = L.hc_mix[q]; o.out = L.hc_out[q];
  return o;
}

SsmWeights ssm_weights(const StackLayer &L) { return {L.ssm_conv, L.ssm_conv_b, L.dt_bias, L.a_log, L.d}; }

size_t k_seq_stride(const dp_model *m, const StackLayer &L) { return (size_t)m->cfg.max_seq * L.k_cols(); }
size_t v_seq_stride(const dp_model *m, const StackLayer &L) { return (size_t)m->cfg.max_seq * L.v_cols(); }

// attention of `rows` rows whose projections are in s->proj; decode: rows are sequences, else consecutive positions
dpk_attn_params attn_params(dp_model *m, int l, int rows, bool decode, int seq, int start_pos) {
  dp_stack *s = m->stack;
  const StackLayer &L = s->layers[l];
  dpk_attn_params p{};
  p.q = s->q;
  p.num_heads = L.c.heads; p.num_kv_heads = L.c.kv_heads; p.head_dim = L.c.dim; p.v_dim = L.c.vdim;
  p.scale = L.c.scale; p.chunk = L.c.chunk; p.kv_f32 = s->f32;
  const size_t e = s->f32 ? 4 : 2;
  const size_t first = decode ? 0 : (size_t)seq;
  p.k = (const __half *)((const char *)m->kc[l]->dptr + first * k_seq_stride(m, L) * e);
  p.v = (const __half *)((const char *)m->vc[l]->dptr + first * v_seq_stride(m, L) * e);
  p.kv_batch_stride = k_seq_stride(m, L); p.v_batch_stride = v_seq_stride(m, L);
  if (decode) {
    p.batch = rows; p.seq_len = 1; p.kv_len = m->cfg.max_seq; p.causal = 0; p.start_pos = 0; p.kv_lens = m->d_kvlen;
  } else {
    p.batch = 1; p.seq_len = rows; p.kv_len = start_pos + rows; p.causal = 1; p.start_pos = start_pos;
  }
  if (L.c.head_gate) { p.gate = s->proj + L.q_cols() + L.k_cols() + L.v_cols(); p.gate_stride = L.proj.N; }
  return p;
}

dp_status unit_qk(dp_model *m, int l, int rows, const RowMap &map) {
  dp_stack *s = m->stack;
  const StackLayer &L = s->layers[l];
  return dpk_unit_qk_kv(m->ctx, s->proj, L.proj.N, s->q, m->kc[l]->dptr, m->vc[l]->dptr, s->f32, L.c.heads, L.c.kv_heads, L.c.dim, L.c.vdim, L.c.unit_rms_qk != 0,
                        s->cfg.eps, k_seq_stride(m, L), v_seq_stride(m, L), rows, map);
}

GemvBf16 gemv(const Mat &w, const float *x) {
  GemvBf16 p;
  p.w = w.w(); p.N = w.N; p.K = w.K; p.w_stride = w.stride; p.x = x;
  return p;
}

// ---- one decode row (sequence 0) ----
dp_status run_single(dp_model *m) {
  dp_ctx *ctx = m->ctx;
  dp_stack *s = m->stack;
  RowMap map;
  map.pos = m->d_pos;
  const int n_layers = (int)s->layers.size();
  // the stream update of sublayer q of layer l, and u of the sublayer that follows
  auto to_streams = [&](GemvBf16 p, int src, int l, int q) {
    const StackLayer &L = s->layers[l];
    p.end = sub_out(L, q);
    p.streams = s->cfg.streams; p.streams_x = s->x[0]; p.next_u = m->h;
    if (q == 0 && L.c.ff) p.next_in = L.hc_in[1];
    else p.next_in = l + 1 < n_layers ? s->layers[l + 1].hc_in[0] : nullptr;
    return dpk_gemv_bf16(ctx, src, GEMV_DST_STREAMS, p);
  };
  for (int l = 0; l < n_layers; l++) {
    StackLayer &L = s->layers[l];
    GemvBf16 in = gemv(L.proj, m->h);
    in.norm = sub_in(s, L, 0); in.pos = m->d_pos; in.y = s->proj;
    DP_TRY(dpk_gemv_bf16(ctx, GEMV_SRC_NORM, GEMV_DST_PLAIN, in));
    if (L.attention()) {
      dpk_attn_params ap = attn_params(m, l, 1, true, 0, 0);
      int splits = 1;
      dpk_attention_scratch_bytes(ctx, ap, &splits);
      if (L.c.unit_rms_qk && dpk_attention_uses_tc(ctx, ap)) {  // that kernel normalises q and k and appends k and v itself
        ap.fuse.qkv = s->proj; ap.fuse.row_stride = (size_t)L.proj.N; ap.fuse.pos = m->d_pos;
        ap.fuse.kc = (__half *)m->kc[l]->dptr; ap.fuse.vc = (__half *)m->vc[l]->dptr;
        ap.fuse.eps = s->cfg.eps; ap.fuse.nh = L.c.heads; ap.fuse.nkv = L.c.kv_heads;
      } else {
        DP_TRY(unit_qk(m, l, 1, map));
      }
      ap.out = s->mix;
      DP_TRY(dpk_attention_split_only(ctx, ap, (float *)m->attn_scratch->dptr, splits));
      if (splits > 1) {
        GemvBf16 o = gemv(L.o, (const float *)m->attn_scratch->dptr);
        o.gate = ap.gate; o.heads = L.c.heads; o.vdim = L.c.vdim; o.splits = splits;
        DP_TRY(to_streams(o, GEMV_SRC_ATTN, l, 0));
      } else {
        DP_TRY(to_streams(gemv(L.o, s->mix), GEMV_SRC_PLAIN, l, 0));
      }
    } else {
      DP_TRY(dpk_ssm_step(ctx, s->proj, L.proj.N, L.ssm, ssm_weights(L), L.st, s->mix, 1, m->d_pos));
      GemvBf16 o = gemv(L.o, s->mix);
      o.norm.norm_w = L.ssm_norm; o.norm.groups = L.c.norm_groups; o.norm.eps = s->cfg.eps;
      DP_TRY(to_streams(o, GEMV_SRC_NORM, l, 0));
    }
    if (L.c.ff) {
      GemvBf16 g = gemv(L.gateup, m->h);
      g.norm = sub_in(s, L, 1); g.pos = m->d_pos; g.y = s->act_f32;
      g.limit = L.c.ff_limit; g.slope = L.c.ff_slope; g.shift = L.c.ff_shift;
      DP_TRY(dpk_gemv_bf16(ctx, GEMV_SRC_NORM, GEMV_DST_GLU, g));
      DP_TRY(to_streams(gemv(L.down, s->act_f32), GEMV_SRC_PLAIN, l, 1));
    }
  }
  m->h_last = m->h;
  return DP_OK;
}

// ---- several rows ----
dp_status product(dp_model *m, const Mat &w, const void *a, int a_stride, float *c, int rows, const GluOut *glu = nullptr) {
  if (m->stack->f32) return dpk_gemm_bf16w_f32(m->ctx, w.w(), w.stride, (const float *)a, a_stride, c, rows, w.N, w.K, glu);
  return dpk_gemm_bf16_tc(m->ctx, w.w(), w.stride, (const __nv_bfloat16 *)a, a_stride, c, rows, w.N, w.K, glu);
}

int a_stride(const dp_stack *s, int K) { return s->f32 ? K : (int)up((size_t)K, 8); }

dp_status run_rows(dp_model *m, int rows, bool decode, int seq, int start_pos) {
  dp_ctx *ctx = m->ctx;
  dp_stack *s = m->stack;
  const int H = s->cfg.width, n_layers = (int)s->layers.size();
  RowMap map;
  if (decode) map.pos = m->d_pos;
  else { map.start_pos = start_pos; map.seq = seq; }
  int cur = 0;
  const float *y = nullptr;
  SublayerOut end;
  auto boundary = [&](int l, int q) -> dp_status {
    DP_TRY(dpk_stream_boundary(ctx, s->x[cur], s->x[cur ^ 1], y, end, sub_in(s, s->layers[l], q), s->cfg.streams, H, s->a, !s->f32, a_stride(s, H), rows, map));
    if (y) cur ^= 1;
    y = s->y;
    end = sub_out(s->layers[l], q);
    return DP_OK;
  };
  for (int l = 0; l < n_layers; l++) {
    StackLayer &L = s->layers[l];
    DP_TRY(boundary(l, 0));
    DP_TRY(product(m, L.proj, s->a, a_stride(s, H), s->proj, rows));
    const int ks = a_stride(s, L.inner());
    if (L.attention()) {
      DP_TRY(unit_qk(m, l, rows, map));
      dpk_attn_params ap = attn_params(m, l, rows, decode, seq, start_pos);
      if (s->f32) ap.out = (float *)s->a;
      else { ap.out_bf16 = (__nv_bfloat16 *)s->a; ap.out_stride = ks; }
      int splits = 1;
      if (decode) dpk_attention_scratch_bytes(ctx, ap, &splits);
      DP_TRY(dpk_attention_with_scratch(ctx, ap, (float *)m->attn_scratch->dptr, splits));
    } else {
      if (decode) {
        DP_TRY(dpk_ssm_step(ctx, s->proj, L.proj.N, L.ssm, ssm_weights(L), L.st, s->mix, rows, m->d_pos));
      } else {
        const bool chunks = !s->f32 && dpk_ssm_chunk_ok(L.ssm, rows);
        DP_TRY(dpk_ssm_conv(ctx, s->proj, L.proj.N, L.ssm, ssm_weights(L), L.st, s->xbc, chunks, s->dt, rows, map));
        if (chunks)
          DP_TRY(dpk_ssm_chunk(ctx, s->proj, L.proj.N, (const __nv_bfloat16 *)s->xbc, s->dt, L.ssm, ssm_weights(L), L.st, s->mix, rows, map));
        else
          DP_TRY(dpk_ssm_scan(ctx, s->proj, L.proj.N, s->xbc, s->dt, L.ssm, ssm_weights(L), L.st, s->mix, rows, map));
      }
      DP_TRY(dpk_group_norm(ctx, s->mix, L.inner(), L.ssm_norm, L.c.norm_groups, s->cfg.eps, L.inner(), s->a, !s->f32, ks, rows));
    }
    DP_TRY(product(m, L.o, s->a, ks, s->y, rows));
    if (L.c.ff) {
      DP_TRY(boundary(l, 1));
      GluOut g;
      g.dst = s->act; g.stride = L.ff_rows(); g.limit = L.c.ff_limit; g.slope = L.c.ff_slope; g.shift = L.c.ff_shift;
      DP_TRY(product(m, L.gateup, s->a, a_stride(s, H), nullptr, rows, &g));
      DP_TRY(product(m, L.down, s->act, L.ff_rows(), s->y, rows));
    }
  }
  DP_TRY(dpk_stream_sum(ctx, s->x[cur], y, end, s->cfg.streams, H, m->h, rows));
  if (!decode) DP_TRY(dpk_hist_commit(ctx, (const HistEntry *)s->entries->dptr, s->n_entries, s->max_channels, rows, start_pos, seq));
  m->h_last = m->h;
  return DP_OK;
}

const char *tensor_name(int id) {
  static const char *names[DP_T_COUNT] = {"embed", "final norm", "norm1", "norm2", "conv1", "conv2", "hc1 in", "hc1 out", "hc1 mix", "hc2 in", "hc2 out", "hc2 mix",
                                          "q", "k", "v", "head gates", "o", "ssm in", "ssm conv", "ssm conv bias", "ssm dt bias", "ssm A_log", "ssm D", "ssm norm",
                                          "ff gate", "ff up", "ff down"};
  return id >= 0 && id < DP_T_COUNT ? names[id] : "?";
}

dp_status check_layer(dp_ctx *ctx, int i, const dp_layer_cfg &c, int width) {
  DP_CHECK(ctx, c.heads > 0 && c.vdim > 0 && c.ff >= 0, "stack: layer %d has no heads, no value size or a negative feed-forward", i);
  if (c.mixer == DP_MIXER_ATTENTION) {
    DP_CHECK(ctx, c.kv_heads > 0 && c.heads % c.kv_heads == 0, "stack: layer %d: %d heads over %d key/value heads", i, c.heads, c.kv_heads);
    DP_CHECK(ctx, c.dim > 0 && c.dim <= 512 && c.vdim <= 512 && c.chunk >= 0, "stack: layer %d: head sizes %d / %d or chunk %d out of range", i, c.dim, c.vdim, c.chunk);
  } else if (c.mixer == DP_MIXER_MAMBA2) {
    DP_CHECK(ctx, c.groups > 0 && c.heads % c.groups == 0, "stack: layer %d: %d heads over %d groups", i, c.heads, c.groups);
    DP_CHECK(ctx, c.state > 0 && dpk_ssm_state_stride(c.state) > 0, "stack: layer %d: state size %d out of range", i, c.state);
    DP_CHECK(ctx, c.conv_taps > 0 && c.norm_groups > 0 && (c.heads * c.vdim) % c.norm_groups == 0, "stack: layer %d: convolution taps or norm groups", i);
  } else {
    return dp_fail(ctx, DP_ERR_UNSUPPORTED, "stack: layer %d: unknown mixer %d", i, c.mixer);
  }
  (void)width;
  return DP_OK;
}

}  // namespace

extern "C" dp_status dp_model_create_stack(dp_ctx *ctx, const dp_stack_cfg *cfg, const dp_layer_cfg *layers, dp_model **out) {
  if (!ctx || !cfg || !layers || !out) return DP_ERR_INVALID;
  const dp_stack_cfg &c = *cfg;
  DP_CHECK(ctx, c.n_layers > 0 && c.width > 0 && c.vocab > 0 && c.max_seq > 0, "stack: invalid configuration");
  DP_CHECK(ctx, c.streams > 0 && c.streams <= DP_MAX_STREAMS, "stack: %d residual streams (1..%d)", c.streams, DP_MAX_STREAMS);
  DP_CHECK(ctx, c.norm_groups > 0 && c.width % c.norm_groups == 0, "stack: width %d does not split into %d norm groups", c.width, c.norm_groups);
  DP_CHECK(ctx, c.input_taps >= 0 && c.max_batch <= 256 && c.max_rows >= 0, "stack: taps, batch or rows out of range");
  DP_CHECK(ctx, c.act_dtype == DP_BF16 || c.act_dtype == DP_F32, "stack: activations are bf16 or f32");
  for (int i = 0; i < c.n_layers; i++) DP_TRY(check_layer(ctx, i, layers[i], c.width));
  dp_model *m = new dp_model();
  dp_stack *s = m->stack = new dp_stack();
  m->ctx = ctx;
  m->cfg = dp_model_cfg{};
  m->cfg.n_layers = c.n_layers; m->cfg.hidden = c.width; m->cfg.vocab = c.vocab; m->cfg.max_seq = c.max_seq; m->cfg.eps = c.eps;
  m->cfg.max_batch = c.max_batch > 0 ? c.max_batch : 1; m->cfg.tp_size = 1;
  m->vocab_l = c.vocab; m->vocab0 = 0;
  s->cfg = c; s->cfg.max_batch = m->cfg.max_batch;
  s->f32 = c.act_dtype == DP_F32;
  const int B = m->cfg.max_batch;
  int t = c.max_rows > 0 ? c.max_rows : (c.max_seq < 2048 ? c.max_seq : 2048);
  if (t < 2) t = 2;
  m->T = B > t ? B : t;
  m->seq_len.assign(B, 0);
  s->layers.resize(c.n_layers);
  m->kc.assign(c.n_layers, nullptr); m->vc.assign(c.n_layers, nullptr);
  size_t scratch = 256;
  const uint64_t one = 1;
  auto build = [&]() -> dp_status {
    DP_TRY(mat_alloc(m, &s->embed, c.vocab, c.width, "embedding_bf16"));
    s->missing = one << DP_T_EMBED | one << DP_T_FINAL_NORM;
    const size_t e = s->f32 ? 4 : 2;
    for (int l = 0; l < c.n_layers; l++) {
      StackLayer &L = s->layers[l];
      L.c = layers[l];
      L.missing = one << DP_T_NORM1 | one << DP_T_O;
      if (c.input_taps) L.missing |= one << DP_T_CONV1;
      if (c.streams > 1) L.missing |= one << DP_T_HC1_IN | one << DP_T_HC1_OUT | one << DP_T_HC1_MIX;
      if (L.attention()) {
        L.missing |= one << DP_T_Q | one << DP_T_K | one << DP_T_V;
        if (L.c.head_gate) L.missing |= one << DP_T_GATE_HEADS;
        DP_TRY(mat_alloc(m, &L.proj, L.q_cols() + L.k_cols() + L.v_cols() + (L.c.head_gate ? L.c.heads : 0), c.width, "w_qkvg_bf16"));
        DP_TRY(dp_buf_acquire(ctx, (size_t)B * c.max_seq * L.k_cols() * e, "kv_cache_keys", &m->kc[l]));
        DP_TRY(dp_buf_acquire(ctx, (size_t)B * c.max_seq * L.v_cols() * e, "kv_cache_values", &m->vc[l]));
        s->state_bytes += (size_t)B * c.max_seq * (L.k_cols() + L.v_cols()) * e;
        const size_t need = (size_t)B * L.c.heads * 32 * (L.c.vdim + 2) * 4;  // at most 32 splits
        if (need > scratch) scratch = need;
      } else {
        for (int id = DP_T_SSM_IN; id <= DP_T_SSM_NORM; id++) L.missing |= one << id;
        L.ssm = {L.c.heads, L.c.vdim, L.c.state, L.c.groups, L.c.conv_taps, dpk_ssm_state_stride(L.c.state)};
        DP_TRY(mat_alloc(m, &L.proj, L.inner() + L.channels() + L.c.heads, c.width, "w_ssm_in_bf16"));
      }
      DP_TRY(mat_alloc(m, &L.o, c.width, L.inner(), "w_o_bf16"));
      if (L.c.ff) {
        L.missing |= one << DP_T_NORM2 | one << DP_T_FF_GATE | one << DP_T_FF_UP | one << DP_T_FF_DOWN;
        if (c.input_taps) L.missing |= one << DP_T_CONV2;
        if (c.streams > 1) L.missing |= one << DP_T_HC2_IN | one << DP_T_HC2_OUT | one << DP_T_HC2_MIX;
        DP_TRY(mat_alloc(m, &L.gateup, 2 * L.ff_rows(), c.width, "w_gateup_bf16"));
        DP_TRY(mat_alloc(m, &L.down, c.width, L.c.ff, "w_down_bf16"));
      }
    }
    auto carve = [&](dp_buf *buf, const char *label, auto &&fn) -> dp_status {
      Carver count;
      fn(count);
      DP_TRY(dp_buf_acquire(ctx, count.off ? count.off : 256, label, buf));
      DP_TRY(dp_buf_fill(ctx, *buf, 0, 0, (*buf)->bytes));
      Carver place;
      place.base = (char *)(*buf)->dptr;
      fn(place);
      return DP_OK;
    };
    DP_TRY(carve(&s->vectors, "stack_vectors", [&](Carver &k) { carve_vectors(s, k); }));
    DP_TRY(carve(&s->state, "sequence_state", [&](Carver &k) { carve_state(s, k); }));
    s->state_bytes += s->state->bytes;
    DP_TRY(carve(&s->acts, "activations", [&](Carver &k) { carve_acts(m, k); }));
    DP_TRY(dp_buf_acquire(ctx, scratch, "attention_split_partials", &m->attn_scratch));
    // one stream: in = out = 1, mix = 1, the plain residual sum, unless vectors are loaded
    if (c.streams == 1) {
      const float v = 1.0f;
      for (StackLayer &L : s->layers)
        for (int q = 0; q < (L.c.ff ? 2 : 1); q++)
          for (float *p : {L.hc_in[q], L.hc_out[q], L.hc_mix[q]}) DP_TRY(upload_raw(ctx, p, &v, 4));
    }
    std::vector<HistEntry> entries;
    for (StackLayer &L : s->layers) {
      if (c.input_taps > 1)
        for (int q = 0; q < (L.c.ff ? 2 : 1); q++)
          entries.push_back({L.stage[q], L.hist[q], (unsigned long long)c.input_taps * c.width, c.width, c.input_taps});
      if (!L.attention() && L.c.conv_taps > 1)
        entries.push_back({L.st.stage, L.st.hist, (unsigned long long)L.st.hist_seq, L.channels(), L.c.conv_taps});
    }
    s->n_entries = (int)entries.size();
    for (const HistEntry &h : entries) if (h.channels > s->max_channels) s->max_channels = h.channels;
    DP_TRY(dp_buf_acquire(ctx, entries.size() * sizeof(HistEntry) + 256, "history_entries", &s->entries));
    if (!entries.empty()) DP_TRY(dp_buf_upload(ctx, s->entries, entries.data(), 0, entries.size() * sizeof(HistEntry)));
    return dp_model_alloc_runner(m);
  };
  const dp_status st = build();
  if (st != DP_OK) {
    const std::string keep = ctx->err;
    dp_model_destroy(m);
    ctx->err = keep;
    return st;
  }
  m->h_last = m->h;
  *out = m;
  return DP_OK;
}

void dp_stack_destroy(dp_model *m) {
  dp_stack *s = m->stack;
  if (!s) return;
  auto rel = [&](dp_buf b) { if (b) dp_buf_release(m->ctx, b); };
  for (StackLayer &L : s->layers) { rel(L.proj.buf); rel(L.o.buf); rel(L.gateup.buf); rel(L.down.buf); }
  rel(s->embed.buf); rel(s->vectors); rel(s->state); rel(s->acts); rel(s->entries);
  delete s;
  m->stack = nullptr;
}

extern "C" size_t dp_model_state_bytes(dp_model *m) {
  if (!m) return 0;
  if (m->stack) return m->stack->state_bytes;
  size_t n = 0;
  for (dp_buf b : m->kc) n += b ? b->bytes : 0;
  for (dp_buf b : m->vc) n += b ? b->bytes : 0;
  return n;
}

extern "C" dp_status dp_model_load_tensor(dp_model *m, int layer, dp_tensor_id id, const void *host, int rows, int cols) {
  if (!m) return DP_ERR_INVALID;
  dp_ctx *ctx = m->ctx;
  dp_stack *s = m->stack;
  DP_CHECK(ctx, s != nullptr, "loadTensor: the model is not described layer by layer");
  DP_CHECK(ctx, host != nullptr && id >= 0 && id < DP_T_COUNT, "loadTensor: null pointer or unknown tensor %d", (int)id);
  const int H = s->cfg.width, S = s->cfg.streams, taps = s->cfg.input_taps;
  auto expect = [&](int r, int c) -> dp_status {
    if (rows != r || cols != c)
      return dp_fail(ctx, DP_ERR_INVALID, "loadTensor: layer %d: %s expects shape [%d,%d], got [%d,%d]", layer, tensor_name(id), r, c, rows, cols);
    return DP_OK;
  };
  const uint64_t bit = (uint64_t)1 << id;
  if (id == DP_T_EMBED || id == DP_T_FINAL_NORM) {
    if (id == DP_T_EMBED) { DP_TRY(expect(s->cfg.vocab, H)); DP_TRY(mat_upload(ctx, s->embed, 0, host, rows, cols)); }
    else { DP_TRY(expect(1, H)); DP_TRY(upload_raw(ctx, s->final_norm, host, (size_t)H * 2)); }
    s->missing &= ~bit;
    return DP_OK;
  }
  DP_CHECK(ctx, layer >= 0 && layer < (int)s->layers.size(), "loadTensor: layer %d out of range", layer);
  StackLayer &L = s->layers[layer];

  auto vec_bf16 = [&](__nv_bfloat16 *dst, int r, int c) -> dp_status {
    if (!dst) return dp_fail(ctx, DP_ERR_INVALID, "loadTensor: layer %d has no %s", layer, tensor_name(id));
    DP_TRY(expect(r, c));
    return upload_raw(ctx, dst, host, (size_t)r * c * 2);
  };
  auto vec_f32 = [&](float *dst, int r, int c) -> dp_status {
    if (!dst) return dp_fail(ctx, DP_ERR_INVALID, "loadTensor: layer %d has no %s", layer, tensor_name(id));
    DP_TRY(expect(r, c));
    return upload_as_f32(ctx, dst, host, (size_t)r * c);
  };
  auto part = [&](bool present, const Mat &w, int row0, int r, int c) -> dp_status {
    if (!present) return dp_fail(ctx, DP_ERR_INVALID, "loadTensor: layer %d has no %s", layer, tensor_name(id));
    DP_TRY(expect(r, c));
    return mat_upload(ctx, w, row0, host, rows, cols);
  };

  const bool att = L.attention();
  dp_status st = DP_OK;
  switch (id) {
    case DP_T_NORM1: st = vec_bf16(L.norm[0], 1, H); break;
    case DP_T_NORM2: st = vec_bf16(L.norm[1], 1, H); break;
    case DP_T_CONV1: st = vec_bf16(L.conv[0], H, taps); break;
    case DP_T_CONV2: st = vec_bf16(L.conv[1], H, taps); break;
    case DP_T_HC1_IN: st = vec_f32(L.hc_in[0], 1, S); break;
    case DP_T_HC1_OUT: st = vec_f32(L.hc_out[0], 1, S); break;
    case DP_T_HC1_MIX: st = vec_f32(L.hc_mix[0], S, S); break;
    case DP_T_HC2_IN: st = vec_f32(L.hc_in[1], 1, S); break;
    case DP_T_HC2_OUT: st = vec_f32(L.hc_out[1], 1, S); break;
    case DP_T_HC2_MIX: st = vec_f32(L.hc_mix[1], S, S); break;
    case DP_T_Q: st = part(att, L.proj, 0, L.q_cols(), H); break;
    case DP_T_K: st = part(att, L.proj, L.q_cols(), L.k_cols(), H); break;
    case DP_T_V: st = part(att, L.proj, L.q_cols() + L.k_cols(), L.v_cols(), H); break;
    case DP_T_GATE_HEADS: st = part(att && L.c.head_gate, L.proj, L.q_cols() + L.k_cols() + L.v_cols(), L.c.heads, H); break;
    case DP_T_O: st = part(true, L.o, 0, H, L.inner()); break;
    case DP_T_SSM_IN: st = part(!att, L.proj, 0, L.proj.N, H); break;
    case DP_T_SSM_CONV: st = vec_f32(L.ssm_conv, L.channels(), L.c.conv_taps); break;
    case DP_T_SSM_CONV_B: st = vec_f32(L.ssm_conv_b, 1, L.channels()); break;
    case DP_T_SSM_DT_BIAS: st = vec_f32(L.dt_bias, 1, L.c.heads); break;
    case DP_T_SSM_A_LOG: st = vec_f32(L.a_log, 1, L.c.heads); break;
    case DP_T_SSM_D: st = vec_f32(L.d, 1, L.c.heads); break;
    case DP_T_SSM_NORM: st = vec_bf16(L.ssm_norm, 1, L.inner()); break;
    case DP_T_FF_GATE:
    case DP_T_FF_UP:
      DP_CHECK(ctx, L.c.ff > 0, "loadTensor: layer %d has no %s", layer, tensor_name(id));
      DP_TRY(expect(L.c.ff, H));
      st = mat_upload_glu(ctx, L.gateup, id == DP_T_FF_UP, host, rows, cols);
      break;
    case DP_T_FF_DOWN: st = part(L.c.ff > 0, L.down, 0, H, L.c.ff); break;
    default: return dp_fail(ctx, DP_ERR_INVALID, "loadTensor: %s is not a layer's tensor", tensor_name(id));
  }
  if (st == DP_OK) L.missing &= ~bit;
  return st;
}

dp_status dp_stack_ready(dp_model *m) {
  dp_stack *s = m->stack;
  for (int id = 0; id < DP_T_COUNT; id++) {
    if (s->missing >> id & 1) return dp_fail(m->ctx, DP_ERR_STATE, "model: %s has not been loaded", tensor_name(id));
    for (size_t l = 0; l < s->layers.size(); l++)
      if (s->layers[l].missing >> id & 1) return dp_fail(m->ctx, DP_ERR_STATE, "model: layer %d: %s has not been loaded", (int)l, tensor_name(id));
  }
  return DP_OK;
}

dp_status dp_stack_embed(dp_model *m, const int *ids, int rows, bool decode) {
  dp_stack *s = m->stack;
  const bool single = decode && rows == 1;
  return dpk_stream_embed(m->ctx, ids, s->embed.w(), s->embed.stride, s->cfg.embed_scale, s->cfg.streams, s->cfg.width, s->x[0], s->layers[0].hc_in[0],
                          single ? m->h : nullptr, rows);
}

dp_status dp_stack_run_layers(dp_model *m, int rows, bool decode, int seq, int start_pos) {
  if (decode && rows == 1) return run_single(m);
  return run_rows(m, rows, decode, seq, start_pos);
}

// final norm and tied head of `rows` rows -> m->logits
dp_status dp_stack_logits(dp_model *m, const float *hrow, int rows) {
  dp_stack *s = m->stack;
  if (rows == 1) {
    GemvBf16 p = gemv(s->embed, hrow);
    p.norm.norm_w = s->final_norm; p.norm.groups = s->cfg.norm_groups; p.norm.eps = s->cfg.eps;
    p.y = m->logits;
    return dpk_gemv_bf16(m->ctx, GEMV_SRC_NORM, GEMV_DST_PLAIN, p);
  }
  const int st = a_stride(s, s->cfg.width);
  DP_TRY(dpk_group_norm(m->ctx, hrow, s->cfg.width, s->final_norm, s->cfg.norm_groups, s->cfg.eps, s->cfg.width, s->a, !s->f32, st, rows));
  return product(m, s->embed, s->a, st, m->logits, rows);
}
