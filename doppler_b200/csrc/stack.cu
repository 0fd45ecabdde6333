// Decoders described layer by layer: weights, per-sequence state and the schedule of their layers.
//
// A dp_model whose `stack` is set is run by the same runner as the dense Q4_K decoder (model.cu: portions, decode
// graph, greedy pick, sequence lengths); this file supplies what differs.  Two schedules:
//
//   one decode row     every kernel rebuilds its own input (gemv_bf16.cu), three kernels for a Mamba-2 sublayer
//                      (projection [norm + input convolution] -> step -> output projection [group norm; streams]),
//                      three for an attention sublayer, two for the feed-forward
//                      (where sublayers have a norm behind them, the residual sum waits for the whole of their result: the
//                      output projection stores it plainly and the next kernel's prologue adds it); lightning: projection ->
//                      step -> output projection [norm, gate]; delta rule: the same three; latent attention: projection ->
//                      queries [norm] -> absorbed queries and cache row -> attention -> values [split merge] -> output
//   several rows       (portions of a prompt, batched decode) one boundary kernel between two sublayers
//                      (streams.cu), tensor-core products, and the mixers' own kernels
//
// A layer may use another one's tensors: it then is a copy of that layer's description with a state of its own.
//
// State of a sequence: K/V or latent rows of the attention layers (contiguous, position p at row p), the recurrent state of
// the recurrent layers, and short histories (rings of `taps` positions) of every causal convolution.  None of it is
// read at or beyond the sequence's length, and position 0 starts from zeros, so a slot is reused by setting its
// length to 0.  A portion leaves the last rows of its histories in a stage; one kernel at its end moves them into the
// rings (writing them earlier would overwrite rows other CTAs of the portion still read).
#include "layers.h"
#include "model.h"

#include <cmath>
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
  // proj: q | k | v | head gates (attention), the Mamba-2 input projection, gate | v | k | q (lightning), q | k | v | b | a1 | g1
  // (delta rule), dq | dkv | head gates (latent attention)
  Mat proj, o, gateup, down;
  Mat a2, g2;      // delta rule: second matrices of decay and gate
  Mat uq, uk, uv;  // latent attention
  Mat ukv;         // latent attention: uk and uv together in f16, heads padded to eight rows (bf16 mode)
  bool up_exact = true;  // every value fits f16
  __nv_bfloat16 *norm[2] = {}, *conv[2] = {}, *post[2] = {}, *mix_norm = nullptr, *dq_norm = nullptr, *dkv_norm = nullptr;
  float *hc_in[2] = {}, *hc_out[2] = {}, *hc_mix[2] = {};
  float *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *d = nullptr;
  float *rate = nullptr;   // Mamba-2, lightning: decay exponent per unit step [heads]; delta rule: exp(A_log) of each key channel
  float *decay = nullptr;  // lightning
  float *hist[2] = {}, *stage[2] = {};
  SsmShape ssm = {};
  DeltaShape delta = {};
  LatentShape lat = {};
  Rotation rot;
  SsmState st;
  uint64_t missing = 0;  // bit per dp_tensor_id still to be loaded
  int owner = -1;        // the layer whose tensors this one uses (-1: its own)
  bool attention() const { return c.mixer == DP_MIXER_ATTENTION; }
  bool mamba() const { return c.mixer == DP_MIXER_MAMBA2; }
  bool lightning() const { return c.mixer == DP_MIXER_LIGHTNING; }
  bool is_delta() const { return c.mixer == DP_MIXER_DELTA; }
  bool latent() const { return c.mixer == DP_MIXER_LATENT; }
  int subs() const { return c.ff ? 2 : 1; }
  int q_cols() const { return c.heads * c.dim; }
  int k_cols() const { return c.kv_heads * c.dim; }
  int v_cols() const { return c.kv_heads * c.vdim; }
  int inner() const { return c.heads * c.vdim; }
  int channels() const { return is_delta() ? delta.channels() : inner() + 2 * ssm.groups * ssm.state; }  // of the recurrence's convolutions
  int ff_rows() const { return (int)up((size_t)c.ff, 8); }
};

}  // namespace

struct RopeTable {
  int dims = 0;
  double base = 0.0;
  dp_buf buf = nullptr;  // cos [max_seq][dims / 2], then sin
};

struct dp_stack {
  dp_stack_cfg cfg;
  bool f32 = false;
  std::vector<StackLayer> layers;
  dp_buf expanded = nullptr;   // latent attention: keys and values of a sequence's tokens, [token][ukv.N] f16

  Mat embed;
  __nv_bfloat16 *final_norm = nullptr;
  uint64_t missing = 0;
  dp_buf vectors = nullptr, state = nullptr, acts = nullptr, entries = nullptr;
  int n_entries = 0, max_channels = 0;
  size_t state_bytes = 0;
  float *x[2], *y, *proj, *q, *xbc, *dt, *mix, *act_f32;
  DeltaRows dl;                // delta rule: a portion's rows (g is written by the decay's product)
  float *dl_g, *gate;          // decays; output gates before their sigmoid
  float *q_abs, *ctx;          // latent attention: absorbed queries, means of the latents
  std::vector<RopeTable> ropes;
  int pending = -1;            // one decode row: s->x[pending] still lacks the last sublayer's result (-1: complete)
  SublayerOut pending_end;
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

// bf16 rows of all heads into a matrix of f16, a head's rows padded to whole groups of eight; *exact is cleared where a value
// does not fit
dp_status mat_upload_f16(dp_ctx *ctx, const Mat &t, int row0, const void *host, int heads, int rows, int cols, bool *exact) {
  const size_t padded = up((size_t)rows, 8);
  std::vector<__half> stage(heads * padded * t.stride, __half(0.0f));
  for (int h = 0; h < heads; h++)
    for (int r = 0; r < rows; r++)
      for (int c = 0; c < cols; c++) {
        const uint32_t bits = (uint32_t)((const uint16_t *)host)[((size_t)h * rows + r) * cols + c] << 16;
        float v;
        memcpy(&v, &bits, 4);
        if (!(fabsf(v) <= 65504.0f)) *exact = false;
        stage[(h * padded + r) * t.stride + c] = __float2half_rn(v);
      }
  DP_CUDA(ctx, cudaMemcpyAsync((char *)t.buf->dptr + (size_t)row0 * t.stride * 2, stage.data(), stage.size() * 2, cudaMemcpyHostToDevice, ctx->stream));
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
    if (L.owner >= 0) continue;
    for (int q = 0; q < L.subs(); q++) {
      c.take(&L.norm[q], H);
      if (taps) c.take(&L.conv[q], H * taps);
      if (s->cfg.post_norm) c.take(&L.post[q], H);
      c.take(&L.hc_in[q], S); c.take(&L.hc_out[q], S); c.take(&L.hc_mix[q], S * S);
    }
    const size_t heads = L.c.heads;
    if (L.mamba()) {
      c.take(&L.conv_w, (size_t)L.channels() * L.c.conv_taps); c.take(&L.conv_b, L.channels());
      c.take(&L.dt_bias, heads); c.take(&L.rate, heads); c.take(&L.d, heads);
      c.take(&L.mix_norm, L.inner());
    } else if (L.lightning()) {
      c.take(&L.rate, heads); c.take(&L.decay, heads); c.take(&L.mix_norm, L.inner());
    } else if (L.is_delta()) {
      c.take(&L.conv_w, (size_t)L.channels() * L.c.conv_taps);
      c.take(&L.rate, heads * L.c.dim); c.take(&L.dt_bias, heads * L.c.dim);
      c.take(&L.mix_norm, L.c.vdim);
    } else if (L.latent()) {
      c.take(&L.dq_norm, L.c.q_rank); c.take(&L.dkv_norm, L.c.kv_rank);
    }
  }
}

void carve_state(dp_stack *s, Carver &c) {
  const size_t H = s->cfg.width, B = s->cfg.max_batch, taps = s->cfg.input_taps;
  for (StackLayer &L : s->layers) {
    if (taps > 1)
      for (int q = 0; q < L.subs(); q++) { c.take(&L.hist[q], B * taps * H); c.take(&L.stage[q], taps * H); }
    if (L.mamba() || L.lightning() || L.is_delta()) {
      L.st.hist_seq = L.lightning() ? 0 : (size_t)L.c.conv_taps * L.channels();
      L.st.s_seq = (size_t)L.inner() * (L.is_delta() ? L.delta.state_stride : L.ssm.state_stride);
      c.take(&L.st.hist, B * L.st.hist_seq); c.take(&L.st.stage, L.st.hist_seq); c.take(&L.st.s, B * L.st.s_seq);
    }
  }
}

void carve_acts(dp_model *m, Carver &c) {
  dp_stack *s = m->stack;
  const size_t T = m->T, H = s->cfg.width, S = s->cfg.streams;
  size_t proj = 0, q = 1, xbc = 1, heads = 1, mix = 1, k = up(H, 8), ff = 1;
  size_t dl_qk = 0, dl_heads = 0, dl_inner = 0, dl_hd = 0, low_a = 0, low_g = 0, records = 0, q_abs = 0, ctx = 0;
  auto most = [](size_t &a, size_t b) { if (b > a) a = b; };
  for (const StackLayer &L : s->layers) {
    most(proj, L.proj.N);
    most(k, L.o.stride);
    most(mix, L.inner());
    if (L.c.ff) most(ff, L.ff_rows());
    if (L.attention()) most(q, L.q_cols());
    if (L.mamba() || L.lightning()) { most(xbc, L.channels()); most(heads, L.c.heads); }
    if (L.is_delta()) {
      most(dl_qk, L.delta.qk()); most(dl_heads, L.c.heads); most(dl_inner, L.inner()); most(dl_hd, (size_t)L.c.heads * L.c.dim);
      most(low_a, L.a2.stride); most(low_g, L.g2.stride); most(records, dpk_delta_record_floats(L.delta, (int)T));
    }
    if (L.latent()) {
      most(q, L.uq.N); most(k, L.uq.stride);
      most(q_abs, (size_t)L.c.heads * L.lat.cols()); most(ctx, (size_t)L.c.heads * L.lat.c_pad());
    }
  }
  c.take(&s->x[0], T * S * H); c.take(&s->x[1], T * S * H); c.take(&s->y, T * H); c.take(&m->h, T * H);
  c.take(&s->proj, T * proj); c.take(&s->q, T * q); c.take(&s->xbc, T * xbc); c.take(&s->dt, T * heads); c.take(&s->mix, T * mix);
  c.take(&s->dl.q, T * dl_qk); c.take(&s->dl.k, T * dl_qk); c.take(&s->dl.beta, T * dl_heads);
  c.take(&s->dl.v, T * dl_inner); c.take(&s->gate, T * dl_inner); c.take(&s->dl_g, T * dl_hd);
  c.take(&s->dl.records, records);
  c.take(&s->dl.a_low, T * low_a); c.take(&s->dl.g_low, T * low_g);
  c.take(&s->q_abs, T * q_abs); c.take(&s->ctx, T * ctx);
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

SublayerOut sub_out(const dp_stack *s, const StackLayer &L, int q) {
  SublayerOut o;
  o.mix = L.hc_mix[q]; o.out = L.hc_out[q];
  o.norm_w = L.post[q]; o.groups = s->cfg.norm_groups; o.eps = s->cfg.eps;
  return o;
}

SsmWeights ssm_weights(const StackLayer &L) {
  SsmWeights w;
  w.conv = L.conv_w; w.conv_b = L.conv_b; w.dt_bias = L.dt_bias; w.a = L.rate; w.d = L.d; w.decay = L.decay;
  return w;
}

DeltaWeights delta_weights(const StackLayer &L) {
  DeltaWeights w;
  w.conv = L.conv_w; w.rate = L.rate; w.bias = L.dt_bias;
  w.a2 = L.a2.w(); w.a2_stride = L.a2.stride; w.g2 = L.g2.w(); w.g2_stride = L.g2.stride;
  return w;
}

// norm of a recurrence's output and, where it has one, the gate behind it
GroupNorm mix_norm(const dp_stack *s, const StackLayer &L) {
  GroupNorm n;
  n.w = L.mix_norm; n.eps = s->cfg.eps;
  if (L.mamba()) n.groups = L.c.norm_groups;
  if (L.lightning()) { n.gate = s->proj; n.gate_stride = L.proj.N; }
  if (L.is_delta()) { n.groups = L.c.heads; n.w_shared = true; n.gate = s->gate; n.gate_stride = L.inner(); }
  return n;
}

LatentCache latent_cache(const dp_model *m, int l) {
  LatentCache c;
  c.rows = m->kc[l]->dptr; c.f32 = m->stack->f32; c.seq = (size_t)m->cfg.max_seq * m->stack->layers[l].lat.cols();
  return c;
}

size_t k_seq_stride(const dp_model *m, const StackLayer &L) { return (size_t)m->cfg.max_seq * L.k_cols(); }
size_t v_seq_stride(const dp_model *m, const StackLayer &L) { return (size_t)m->cfg.max_seq * L.v_cols(); }

// attention of `rows` rows whose projections are in s->proj; decode: rows are sequences, else consecutive positions
dpk_attn_params attn_params(dp_model *m, int l, int rows, bool decode, int seq, int start_pos) {
  dp_stack *s = m->stack;
  const StackLayer &L = s->layers[l];
  dpk_attn_params p{};
  p.q = s->q;
  p.scale = L.c.scale; p.chunk = L.c.chunk; p.kv_f32 = s->f32;
  const size_t e = s->f32 ? 4 : 2;
  const size_t first = decode ? 0 : (size_t)seq;
  if (L.latent()) {  // absorbed queries on the cache rows: one key/value head, values are the first part of the keys
    const LatentCache cache = latent_cache(m, l);
    p.q = s->q_abs;
    p.num_heads = L.c.heads; p.num_kv_heads = 1; p.head_dim = L.lat.cols(); p.v_dim = L.lat.c_pad(); p.v_row_stride = L.lat.cols();
    p.k = p.v = (const __half *)((const char *)cache.rows + first * cache.seq * e);
    p.kv_batch_stride = p.v_batch_stride = cache.seq;
  } else {
    p.num_heads = L.c.heads; p.num_kv_heads = L.c.kv_heads; p.head_dim = L.c.dim; p.v_dim = L.c.vdim;
    p.k = (const __half *)((const char *)m->kc[l]->dptr + first * k_seq_stride(m, L) * e);
    p.v = (const __half *)((const char *)m->vc[l]->dptr + first * v_seq_stride(m, L) * e);
    p.kv_batch_stride = k_seq_stride(m, L); p.v_batch_stride = v_seq_stride(m, L);
  }
  if (decode) {
    p.batch = rows; p.seq_len = 1; p.kv_len = m->cfg.max_seq; p.causal = 0; p.start_pos = 0; p.kv_lens = m->d_kvlen;
  } else {
    p.batch = 1; p.seq_len = rows; p.kv_len = start_pos + rows; p.causal = 1; p.start_pos = start_pos;
  }
  if (L.c.head_gate && L.attention()) { p.gate = s->proj + L.q_cols() + L.k_cols() + L.v_cols(); p.gate_stride = L.proj.N; }
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
  const bool post = s->cfg.post_norm != 0;
  int cur = 0;            // post: where the residual row is
  bool waiting = false;   // post: s->y still has to be added to it
  SublayerOut end;
  // the first product of sublayer q of layer l, from the normed residual
  auto enter = [&](GemvBf16 p, int dst, int l, int q) -> dp_status {
    p.norm = sub_in(s, s->layers[l], q);
    p.pos = m->d_pos;
    if (!post) { p.x = m->h; return dpk_gemv_bf16(ctx, GEMV_SRC_NORM, dst, p); }
    p.x = s->x[cur];
    if (!waiting) return dpk_gemv_bf16(ctx, GEMV_SRC_NORM, dst, p);
    p.res = end; p.res_y = s->y; p.x_out = s->x[cur ^ 1];
    cur ^= 1;
    waiting = false;
    return dpk_gemv_bf16(ctx, GEMV_SRC_RESIDUAL, dst, p);
  };
  // the last product of sublayer q of layer l: the stream update, and u of the sublayer that follows
  auto leave = [&](GemvBf16 p, int src, int l, int q) -> dp_status {
    const StackLayer &L = s->layers[l];
    if (post) {
      p.y = s->y;
      end = sub_out(s, L, q);
      waiting = true;
      return dpk_gemv_bf16(ctx, src, GEMV_DST_PLAIN, p);
    }
    if (src == GEMV_SRC_GATED) return dp_fail(ctx, DP_ERR_UNSUPPORTED, "stack: gated recurrences come with norms behind the sublayers");
    p.end = sub_out(s, L, q);
    p.streams = s->cfg.streams; p.streams_x = s->x[0]; p.next_u = m->h;
    if (q == 0 && L.c.ff) p.next_in = L.hc_in[1];
    else p.next_in = l + 1 < n_layers ? s->layers[l + 1].hc_in[0] : nullptr;
    return dpk_gemv_bf16(ctx, src, GEMV_DST_STREAMS, p);
  };
  for (int l = 0; l < n_layers; l++) {
    StackLayer &L = s->layers[l];
    GemvBf16 in = gemv(L.proj, nullptr);
    in.y = s->proj;
    DP_TRY(enter(in, GEMV_DST_PLAIN, l, 0));
    if (L.attention() || L.latent()) {
      if (L.latent()) {
        GemvBf16 uq = gemv(L.uq, s->proj);
        uq.norm.norm_w = L.dq_norm; uq.norm.eps = s->cfg.eps; uq.y = s->q;
        DP_TRY(dpk_gemv_bf16(ctx, GEMV_SRC_NORM, GEMV_DST_PLAIN, uq));
        DP_TRY(dpk_latent_absorb_step(ctx, s->proj, L.lat, L.dkv_norm, L.rot, latent_cache(m, l), L.uk.w(), L.uk.stride, s->q, s->q_abs, m->d_pos));
      }
      dpk_attn_params ap = attn_params(m, l, 1, true, 0, 0);
      int splits = 1;
      dpk_attention_scratch_bytes(ctx, ap, &splits);
      if (L.attention()) {
        if (L.c.unit_rms_qk && dpk_attention_uses_tc(ctx, ap)) {  // that kernel normalises q and k and appends k and v itself
          ap.fuse.qkv = s->proj; ap.fuse.row_stride = (size_t)L.proj.N; ap.fuse.pos = m->d_pos;
          ap.fuse.kc = (__half *)m->kc[l]->dptr; ap.fuse.vc = (__half *)m->vc[l]->dptr;
          ap.fuse.eps = s->cfg.eps; ap.fuse.nh = L.c.heads; ap.fuse.nkv = L.c.kv_heads;
        } else {
          DP_TRY(unit_qk(m, l, 1, map));
        }
      }
      ap.out = L.latent() ? s->ctx : s->mix;
      DP_TRY(dpk_attention_split_only(ctx, ap, (float *)m->attn_scratch->dptr, splits));
      if (L.latent()) {
        DP_TRY(dpk_latent_values_step(ctx, splits > 1 ? (const float *)m->attn_scratch->dptr : s->ctx, splits, L.lat, L.uv.w(), L.uv.stride,
                                      L.c.head_gate ? s->proj + L.lat.gate_col() : nullptr, s->mix));
        DP_TRY(leave(gemv(L.o, s->mix), GEMV_SRC_PLAIN, l, 0));
      } else if (splits > 1) {
        GemvBf16 o = gemv(L.o, (const float *)m->attn_scratch->dptr);
        o.gate = ap.gate; o.heads = L.c.heads; o.vdim = L.c.vdim; o.splits = splits;
        DP_TRY(leave(o, GEMV_SRC_ATTN, l, 0));
      } else {
        DP_TRY(leave(gemv(L.o, s->mix), GEMV_SRC_PLAIN, l, 0));
      }
    } else {
      if (L.is_delta()) DP_TRY(dpk_delta_step(ctx, s->proj, L.proj.N, L.delta, delta_weights(L), L.st, s->mix, s->gate, 1, m->d_pos));
      else DP_TRY(dpk_ssm_step(ctx, s->proj, L.proj.N, L.ssm, ssm_weights(L), L.st, s->mix, 1, m->d_pos));
      const GroupNorm n = mix_norm(s, L);
      GemvBf16 o = gemv(L.o, s->mix);
      o.norm.norm_w = n.w; o.norm.groups = n.groups; o.norm.eps = n.eps;
      o.gate = n.gate; o.norm_w_shared = n.w_shared;
      DP_TRY(leave(o, n.gate ? GEMV_SRC_GATED : GEMV_SRC_NORM, l, 0));
    }
    if (L.c.ff) {
      GemvBf16 g = gemv(L.gateup, nullptr);
      g.y = s->act_f32;
      g.limit = L.c.ff_limit; g.slope = L.c.ff_slope; g.shift = L.c.ff_shift;
      DP_TRY(enter(g, GEMV_DST_GLU, l, 1));
      DP_TRY(leave(gemv(L.down, s->act_f32), GEMV_SRC_PLAIN, l, 1));
    }
  }
  s->pending = post ? cur : -1;
  s->pending_end = end;
  m->h_last = m->h;
  return DP_OK;
}

// ---- several rows ----
dp_status product(dp_model *m, const Mat &w, const void *a, int a_stride, float *c, int rows, const GluOut *glu = nullptr, const DecayOut *decay = nullptr) {
  if (m->stack->f32) return dpk_gemm_bf16w_f32(m->ctx, w.w(), w.stride, (const float *)a, a_stride, c, rows, w.N, w.K, glu, decay);
  return dpk_gemm_bf16_tc(m->ctx, w.w(), w.stride, (const __nv_bfloat16 *)a, a_stride, c, rows, w.N, w.K, glu, decay);
}

int a_stride(const dp_stack *s, int K) { return s->f32 ? K : (int)up((size_t)K, 8); }

// The delta rule over a portion: s->proj -> s->mix and s->gate.
dp_status delta_portion(dp_model *m, StackLayer &L, int rows, const RowMap &map) {
  dp_stack *s = m->stack;
  DeltaRows r = s->dl;
  r.g = s->dl_g;
  r.a_low_stride = L.a2.stride; r.g_low_stride = L.g2.stride;
  if (s->f32) r.a_low = r.g_low = nullptr;  // the products read the projections themselves
  DP_TRY(dpk_delta_rows(m->ctx, s->proj, L.proj.N, L.delta, delta_weights(L), L.st, r, rows, map));
  DecayOut decay;
  decay.rate = L.rate; decay.bias = L.dt_bias;
  if (s->f32) {
    DP_TRY(product(m, L.a2, s->proj + L.delta.a1_col(), L.proj.N, s->dl_g, rows, nullptr, &decay));
    DP_TRY(product(m, L.g2, s->proj + L.delta.g1_col(), L.proj.N, s->gate, rows));
  } else {
    DP_TRY(product(m, L.a2, r.a_low, r.a_low_stride, s->dl_g, rows, nullptr, &decay));
    DP_TRY(product(m, L.g2, r.g_low, r.g_low_stride, s->gate, rows));
  }
  return dpk_delta_scan(m->ctx, L.delta, L.st, r, s->mix, rows, map);
}

// Keys and values of all heads formed from the cached latents (portions of many rows): what `expanded` must be able to hold,
// and where it pays: forming them costs as much per token as `rows` queries save against the absorbed form, whose products
// run at about a quarter of the rate.
bool expand_pays(const dp_stack *s, const StackLayer &L, int rows, int kv_len) {
  const LatentShape &sh = L.lat;
  if (s->f32 || !s->expanded || !L.up_exact || rows < 16 || (size_t)kv_len * L.ukv.N * 2 > s->expanded->bytes) return false;
  const long saved = 2l * sh.kv_rank + sh.rot_dim - (sh.dim + sh.rot_dim + sh.vdim);
  return saved > 0 ? saved * 4 * rows >= (long)sh.kv_rank * (sh.dim + sh.vdim) : true;
}

dp_status latent_expanded(dp_model *m, int l, int rows, int seq, int start_pos, int ks) {
  dp_stack *s = m->stack;
  StackLayer &L = s->layers[l];
  const LatentShape &sh = L.lat;
  const LatentCache cache = latent_cache(m, l);
  const int kv_len = start_pos + rows, N = L.ukv.N;
  const __half *lat = (const __half *)cache.rows + (size_t)seq * cache.seq;
  __half *kv = (__half *)s->expanded->dptr;
  DP_TRY(dpk_gemm_f16_tc(m->ctx, (const __half *)L.ukv.w(), L.ukv.stride, lat, sh.cols(), kv, N, kv_len, N, sh.kv_rank));
  dpk_attn_params p{};
  p.q = s->q;
  p.scale = L.c.scale;
  p.num_heads = p.num_kv_heads = sh.heads; p.head_dim = sh.dim + sh.rot_dim; p.v_dim = sh.vdim;
  p.k = kv; p.k_dim = sh.dim; p.k_row_stride = N;
  p.v = kv + (size_t)sh.heads * up(sh.dim, 8); p.v_row_stride = N;
  p.k2 = lat + sh.c_pad(); p.k2_dim = sh.rot_dim; p.k2_row_stride = sh.cols();
  p.batch = 1; p.seq_len = rows; p.kv_len = kv_len; p.causal = 1; p.start_pos = start_pos;
  p.out_bf16 = (__nv_bfloat16 *)s->a; p.out_stride = ks;
  if (L.c.head_gate) { p.gate = s->proj + sh.gate_col(); p.gate_stride = L.proj.N; }
  return dpk_attention_with_scratch(m->ctx, p, nullptr, 1);
}

// Latent attention of several rows: s->proj -> head outputs in s->a (rows of `ks` elements).
dp_status latent_rows(dp_model *m, int l, int rows, bool decode, int seq, int start_pos, int ks, const RowMap &map) {
  dp_ctx *ctx = m->ctx;
  dp_stack *s = m->stack;
  StackLayer &L = s->layers[l];
  const LatentShape &sh = L.lat;
  GroupNorm n;
  n.w = L.dq_norm; n.eps = s->cfg.eps;
  const int qs = a_stride(s, L.uq.K);
  DP_TRY(dpk_group_norm(ctx, s->proj, L.proj.N, n, sh.q_rank, s->a, !s->f32, qs, rows));
  DP_TRY(product(m, L.uq, s->a, qs, s->q, rows));
  const bool expand = !decode && expand_pays(s, L, rows, start_pos + rows);
  DP_TRY(dpk_latent_append(ctx, s->proj, L.proj.N, sh, L.dkv_norm, L.rot, latent_cache(m, l), s->q, expand ? nullptr : s->q_abs, rows, map));
  if (expand) return latent_expanded(m, l, rows, seq, start_pos, ks);
  GroupedProduct p;
  p.w = L.uk.w(); p.w_z = (size_t)sh.dim * L.uk.stride; p.w_n = 1; p.w_k = L.uk.stride;
  p.x = s->q; p.x_row = L.uq.N; p.x_z = sh.dim + sh.rot_dim;
  p.y = s->q_abs; p.y_row = (size_t)sh.heads * sh.cols(); p.y_z = sh.cols();
  p.rows = rows; p.heads = sh.heads; p.N = sh.kv_rank; p.K = sh.dim;
  DP_TRY(dpk_grouped_product(ctx, p));
  dpk_attn_params ap = attn_params(m, l, rows, decode, seq, start_pos);
  ap.out = s->ctx;
  int splits = 1;
  if (dpk_attention_scratch_bytes(ctx, ap, &splits) > m->attn_scratch->bytes) splits = 1;
  DP_TRY(dpk_attention_with_scratch(ctx, ap, (float *)m->attn_scratch->dptr, splits));
  p = GroupedProduct();
  p.w = L.uv.w(); p.w_z = (size_t)sh.vdim * L.uv.stride; p.w_n = L.uv.stride; p.w_k = 1;
  p.x = s->ctx; p.x_row = (size_t)sh.heads * sh.c_pad(); p.x_z = sh.c_pad();
  p.y = s->a; p.y_bf16 = !s->f32; p.y_row = ks; p.y_z = sh.vdim;
  if (L.c.head_gate) { p.gate = s->proj + sh.gate_col(); p.gate_stride = L.proj.N; }
  p.rows = rows; p.heads = sh.heads; p.N = sh.vdim; p.K = sh.kv_rank;
  return dpk_grouped_product(ctx, p);
}

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
  s->pending = -1;
  auto boundary = [&](int l, int q) -> dp_status {
    DP_TRY(dpk_stream_boundary(ctx, s->x[cur], s->x[cur ^ 1], y, end, sub_in(s, s->layers[l], q), s->cfg.streams, H, s->a, !s->f32, a_stride(s, H), rows, map));
    if (y) cur ^= 1;
    y = s->y;
    end = sub_out(s, s->layers[l], q);
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
    } else if (L.latent()) {
      DP_TRY(latent_rows(m, l, rows, decode, seq, start_pos, ks, map));
    } else {
      if (L.is_delta()) {
        if (decode) DP_TRY(dpk_delta_step(ctx, s->proj, L.proj.N, L.delta, delta_weights(L), L.st, s->mix, s->gate, rows, m->d_pos));
        else DP_TRY(delta_portion(m, L, rows, map));
      } else if (decode) {
        DP_TRY(dpk_ssm_step(ctx, s->proj, L.proj.N, L.ssm, ssm_weights(L), L.st, s->mix, rows, m->d_pos));
      } else {
        const bool chunks = !s->f32 && dpk_ssm_chunk_ok(L.ssm, rows);
        DP_TRY(dpk_ssm_conv(ctx, s->proj, L.proj.N, L.ssm, ssm_weights(L), L.st, s->xbc, chunks, s->dt, rows, map));
        if (chunks)
          DP_TRY(dpk_ssm_chunk(ctx, s->proj, L.proj.N, (const __nv_bfloat16 *)s->xbc, s->dt, L.ssm, ssm_weights(L), L.st, s->mix, rows, map));
        else
          DP_TRY(dpk_ssm_scan(ctx, s->proj, L.proj.N, s->xbc, s->dt, L.ssm, ssm_weights(L), L.st, s->mix, rows, map));
      }
      DP_TRY(dpk_group_norm(ctx, s->mix, L.inner(), mix_norm(s, L), L.inner(), s->a, !s->f32, ks, rows));
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
                                          "ff gate", "ff up", "ff down", "norm1b", "norm2b", "gate", "mixer norm", "q conv", "k conv", "v conv", "b", "a1", "a2",
                                          "g1", "g2", "A_log", "dt_bias", "dq", "dq norm", "uq", "dkv", "dkv norm", "uk", "uv"};
  return id >= 0 && id < DP_T_COUNT ? names[id] : "?";
}

dp_status check_layer(dp_ctx *ctx, int i, const dp_layer_cfg &c, const dp_stack_cfg &stack) {
  DP_CHECK(ctx, c.heads > 0 && c.vdim > 0 && c.ff >= 0, "stack: layer %d has no heads, no value size or a negative feed-forward", i);
  if (c.mixer == DP_MIXER_ATTENTION) {
    DP_CHECK(ctx, c.kv_heads > 0 && c.heads % c.kv_heads == 0, "stack: layer %d: %d heads over %d key/value heads", i, c.heads, c.kv_heads);
    DP_CHECK(ctx, c.dim > 0 && c.dim <= 512 && c.vdim <= 512 && c.chunk >= 0, "stack: layer %d: head sizes %d / %d or chunk %d out of range", i, c.dim, c.vdim, c.chunk);
  } else if (c.mixer == DP_MIXER_MAMBA2) {
    DP_CHECK(ctx, c.groups > 0 && c.heads % c.groups == 0, "stack: layer %d: %d heads over %d groups", i, c.heads, c.groups);
    DP_CHECK(ctx, c.state > 0 && dpk_ssm_state_stride(c.state) > 0, "stack: layer %d: state size %d out of range", i, c.state);
    DP_CHECK(ctx, c.conv_taps > 0 && c.norm_groups > 0 && (c.heads * c.vdim) % c.norm_groups == 0, "stack: layer %d: convolution taps or norm groups", i);
  } else if (c.mixer == DP_MIXER_LIGHTNING) {
    DP_CHECK(ctx, c.dim > 0 && dpk_ssm_state_stride(c.dim) > 0 && c.decay, "stack: layer %d: key size %d out of range or no decays", i, c.dim);
    for (int h = 0; h < c.heads; h++) DP_CHECK(ctx, c.decay[h] >= 0.0 && c.decay[h] <= 1.0, "stack: layer %d: decay of head %d outside [0, 1]", i, h);
  } else if (c.mixer == DP_MIXER_DELTA) {
    DP_CHECK(ctx, c.kv_heads > 0 && c.heads % c.kv_heads == 0, "stack: layer %d: %d heads over %d key/value heads", i, c.heads, c.kv_heads);
    DP_CHECK(ctx, c.dim > 0 && dpk_ssm_state_stride(c.dim) > 0, "stack: layer %d: key size %d out of range", i, c.dim);
    DP_CHECK(ctx, c.conv_taps > 0 && c.decay_rank > 0 && c.gate_rank > 0, "stack: layer %d: convolution taps or low-rank sizes", i);
  } else if (c.mixer == DP_MIXER_LATENT) {
    DP_CHECK(ctx, c.dim > 0 && c.q_rank > 0 && c.kv_rank > 0 && c.rot_dim > 0 && c.rot_dim % 2 == 0 && c.rot_base > 0.0, "stack: layer %d: latent attention sizes", i);
    DP_CHECK(ctx, c.kv_rank + c.rot_dim <= 976 && c.vdim <= 512 && c.chunk == 0, "stack: layer %d: latent of %d + %d values or value size %d out of range", i, c.kv_rank,
             c.rot_dim, c.vdim);
  } else {
    return dp_fail(ctx, DP_ERR_UNSUPPORTED, "stack: layer %d: unknown mixer %d", i, c.mixer);
  }
  DP_CHECK(ctx, (c.mixer != DP_MIXER_LIGHTNING && c.mixer != DP_MIXER_DELTA) || stack.post_norm, "stack: layer %d: this mixer comes with norms behind the sublayers", i);
  return DP_OK;
}

// a layer that uses another one's tensors must be described like it
bool same_layer(const dp_layer_cfg &a, const dp_layer_cfg &b) {
  dp_layer_cfg x = a, y = b;
  x.share = y.share = 0;
  if ((x.decay == nullptr) != (y.decay == nullptr)) return false;
  if (x.decay)
    for (int h = 0; h < a.heads && h < b.heads; h++)
      if (x.decay[h] != y.decay[h]) return false;
  return x.mixer == y.mixer && x.heads == y.heads && x.vdim == y.vdim && x.kv_heads == y.kv_heads && x.dim == y.dim && x.chunk == y.chunk &&
         x.unit_rms_qk == y.unit_rms_qk && x.head_gate == y.head_gate && x.scale == y.scale && x.state == y.state && x.groups == y.groups &&
         x.conv_taps == y.conv_taps && x.norm_groups == y.norm_groups && x.ff == y.ff && x.ff_limit == y.ff_limit && x.ff_slope == y.ff_slope &&
         x.ff_shift == y.ff_shift && x.decay_rank == y.decay_rank && x.gate_rank == y.gate_rank && x.q_rank == y.q_rank && x.kv_rank == y.kv_rank &&
         x.rot_dim == y.rot_dim && x.rot_base == y.rot_base;
}

// cos and sin of every position and pair; angles in double, so a position's error is the rounding of its table entries
dp_status rope_table(dp_model *m, int dims, double base, Rotation *out) {
  dp_stack *s = m->stack;
  const size_t half = dims / 2, n = (size_t)m->cfg.max_seq * half;
  dp_buf buf = nullptr;
  for (const RopeTable &t : s->ropes)
    if (t.dims == dims && t.base == base) buf = t.buf;
  if (!buf) {
    DP_TRY(dp_buf_acquire(m->ctx, 2 * n * 4, "rotation_table", &buf));
    RopeTable t;
    t.dims = dims; t.base = base; t.buf = buf;
    s->ropes.push_back(t);
    std::vector<float> v(2 * n);
    for (size_t i = 0; i < half; i++) {
      const double f = pow(base, -2.0 * (double)i / dims);
      for (size_t p = 0; p < (size_t)m->cfg.max_seq; p++) {
        v[p * half + i] = (float)cos((double)p * f);
        v[n + p * half + i] = (float)sin((double)p * f);
      }
    }
    DP_TRY(dp_buf_upload(m->ctx, buf, v.data(), 0, 2 * n * 4));
  }
  out->cos_t = (const float *)buf->dptr;
  out->sin_t = out->cos_t + n;
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
  DP_CHECK(ctx, !c.post_norm || c.streams == 1, "stack: norms behind the sublayers come with one residual stream");
  DP_CHECK(ctx, c.residual_mult == 0.0f || c.streams == 1, "stack: a residual factor comes with one residual stream");
  for (int i = 0; i < c.n_layers; i++) {
    DP_TRY(check_layer(ctx, i, layers[i], c));
    const int o = layers[i].share - 1;
    DP_CHECK(ctx, o < c.n_layers && o >= -1 && o != i && (o < 0 || (layers[o].share == 0 && same_layer(layers[i], layers[o]))),
             "stack: layer %d cannot use the tensors of layer %d", i, o);
  }
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
    size_t expand_cols = 0;
    auto miss = [](StackLayer &L, std::initializer_list<int> ids) { for (int id : ids) L.missing |= (uint64_t)1 << id; };
    for (int l = 0; l < c.n_layers; l++) {
      StackLayer &L = s->layers[l];
      L.c = layers[l];
      if (L.c.share) { L.owner = L.c.share - 1; continue; }
      miss(L, {DP_T_NORM1, DP_T_O});
      if (c.input_taps) miss(L, {DP_T_CONV1});
      if (c.post_norm) miss(L, {DP_T_NORM1B});
      if (c.streams > 1) miss(L, {DP_T_HC1_IN, DP_T_HC1_OUT, DP_T_HC1_MIX});
      if (L.attention()) {
        miss(L, {DP_T_Q, DP_T_K, DP_T_V});
        if (L.c.head_gate) miss(L, {DP_T_GATE_HEADS});
        DP_TRY(mat_alloc(m, &L.proj, L.q_cols() + L.k_cols() + L.v_cols() + (L.c.head_gate ? L.c.heads : 0), c.width, "w_qkvg_bf16"));
      } else if (L.mamba()) {
        for (int id = DP_T_SSM_IN; id <= DP_T_SSM_NORM; id++) L.missing |= one << id;
        L.ssm = {L.c.heads, L.c.vdim, L.c.state, L.c.groups, L.c.conv_taps, dpk_ssm_state_stride(L.c.state), true};
        DP_TRY(mat_alloc(m, &L.proj, L.inner() + L.channels() + L.c.heads, c.width, "w_ssm_in_bf16"));
      } else if (L.lightning()) {
        miss(L, {DP_T_Q, DP_T_K, DP_T_V, DP_T_GATE, DP_T_MIX_NORM});
        L.ssm = {L.c.heads, L.c.vdim, L.c.dim, L.c.heads, 1, dpk_ssm_state_stride(L.c.dim), false};
        DP_TRY(mat_alloc(m, &L.proj, L.inner() + L.channels(), c.width, "w_gvkq_bf16"));
      } else if (L.is_delta()) {
        miss(L, {DP_T_Q, DP_T_K, DP_T_V, DP_T_CONV_Q, DP_T_CONV_K, DP_T_CONV_V, DP_T_BETA, DP_T_A1, DP_T_A2, DP_T_G1, DP_T_G2, DP_T_A_LOG, DP_T_DT_BIAS, DP_T_MIX_NORM});
        L.delta = {L.c.heads, L.c.kv_heads, L.c.dim, L.c.vdim, L.c.conv_taps, L.c.decay_rank, L.c.gate_rank, dpk_ssm_state_stride(L.c.dim)};
        DP_TRY(mat_alloc(m, &L.proj, L.delta.proj_cols(), c.width, "w_qkvbag_bf16"));
        DP_TRY(mat_alloc(m, &L.a2, L.c.heads * L.c.dim, L.c.decay_rank, "w_a2_bf16"));
        DP_TRY(mat_alloc(m, &L.g2, L.inner(), L.c.gate_rank, "w_g2_bf16"));
      } else {
        miss(L, {DP_T_DQ, DP_T_DQ_NORM, DP_T_UQ, DP_T_DKV, DP_T_DKV_NORM, DP_T_UK, DP_T_UV});
        if (L.c.head_gate) miss(L, {DP_T_GATE_HEADS});
        L.lat = {L.c.heads, L.c.dim, L.c.vdim, L.c.q_rank, L.c.kv_rank, L.c.rot_dim, c.eps, L.c.scale};
        DP_TRY(mat_alloc(m, &L.proj, L.lat.gate_col() + (L.c.head_gate ? L.c.heads : 0), c.width, "w_dq_dkv_g_bf16"));
        DP_TRY(mat_alloc(m, &L.uq, L.c.heads * (L.c.dim + L.c.rot_dim), L.c.q_rank, "w_uq_bf16"));
        DP_TRY(mat_alloc(m, &L.uk, L.c.heads * L.c.dim, L.c.kv_rank, "w_uk_bf16"));
        DP_TRY(mat_alloc(m, &L.uv, L.c.heads * L.c.vdim, L.c.kv_rank, "w_uv_bf16"));
        if (!s->f32) {
          DP_TRY(mat_alloc(m, &L.ukv, (int)(L.c.heads * (up(L.c.dim, 8) + up(L.c.vdim, 8))), L.c.kv_rank, "w_ukv_f16"));
          m->weight_bytes -= (size_t)L.ukv.N * L.ukv.stride * 2;  // a copy; a decode step reads uk and uv
          if (up(L.c.dim, 8) + up(L.c.rot_dim, 8) <= 192 && L.c.vdim <= 128 && (size_t)L.ukv.N > expand_cols) expand_cols = L.ukv.N;
        }
        DP_TRY(rope_table(m, L.c.rot_dim, L.c.rot_base, &L.rot));
      }
      DP_TRY(mat_alloc(m, &L.o, c.width, L.inner(), "w_o_bf16"));
      if (L.c.ff) {
        miss(L, {DP_T_NORM2, DP_T_FF_GATE, DP_T_FF_UP, DP_T_FF_DOWN});
        if (c.input_taps) miss(L, {DP_T_CONV2});
        if (c.post_norm) miss(L, {DP_T_NORM2B});
        if (c.streams > 1) miss(L, {DP_T_HC2_IN, DP_T_HC2_OUT, DP_T_HC2_MIX});
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
    for (int l = 0; l < c.n_layers; l++) {
      const int o = s->layers[l].owner;
      if (o >= 0) {  // the owner's description, weights and vectors, nothing to load
        s->layers[l] = s->layers[o];
        s->layers[l].owner = o;
        s->layers[l].missing = 0;
      }
      StackLayer &L = s->layers[l];
      if (L.attention()) {
        DP_TRY(dp_buf_acquire(ctx, (size_t)B * c.max_seq * L.k_cols() * e, "kv_cache_keys", &m->kc[l]));
        DP_TRY(dp_buf_acquire(ctx, (size_t)B * c.max_seq * L.v_cols() * e, "kv_cache_values", &m->vc[l]));
        s->state_bytes += (size_t)B * c.max_seq * (L.k_cols() + L.v_cols()) * e;
        const size_t need = (size_t)B * L.c.heads * 32 * (L.c.vdim + 2) * 4;  // at most 32 splits
        if (need > scratch) scratch = need;
      } else if (L.latent()) {
        const size_t bytes = (size_t)B * c.max_seq * L.lat.cols() * e;
        DP_TRY(dp_buf_acquire(ctx, bytes, "latent_cache", &m->kc[l]));
        DP_TRY(dp_buf_fill(ctx, m->kc[l], 0, 0, m->kc[l]->bytes));  // the padding of its rows stays zero
        s->state_bytes += bytes;
        // a wave of CTAs beside the rows: short portions split their keys too
        const size_t need = ((size_t)B * 32 + ctx->sm_count + 64) * L.c.heads * (L.lat.c_pad() + 2) * 4;
        if (need > scratch) scratch = need;
      }
    }
    if (expand_cols) {
      const size_t most = (size_t)4 << 30, bytes = (size_t)c.max_seq * expand_cols * 2;  // longer sequences take the absorbed form
      DP_TRY(dp_buf_acquire(ctx, bytes < most ? bytes : most, "latent_expanded", &s->expanded));
    }
    DP_TRY(carve(&s->state, "sequence_state", [&](Carver &k) { carve_state(s, k); }));
    s->state_bytes += s->state->bytes;
    DP_TRY(carve(&s->acts, "activations", [&](Carver &k) { carve_acts(m, k); }));
    DP_TRY(dp_buf_acquire(ctx, scratch, "attention_split_partials", &m->attn_scratch));
    // one stream: in = out = 1, mix = 1, the plain residual sum, unless vectors are loaded
    if (c.streams == 1) {
      const float v = 1.0f, mult = c.residual_mult == 0.0f ? 1.0f : c.residual_mult;
      for (StackLayer &L : s->layers)
        for (int q = 0; q < L.subs() && L.owner < 0; q++) {
          for (float *p : {L.hc_in[q], L.hc_mix[q]}) DP_TRY(upload_raw(ctx, p, &v, 4));
          DP_TRY(upload_raw(ctx, L.hc_out[q], &mult, 4));
        }
    }
    for (StackLayer &L : s->layers)
      if (L.lightning() && L.owner < 0) {
        std::vector<float> a(L.c.heads), d(L.c.heads);
        for (int h = 0; h < L.c.heads; h++) {
          d[h] = (float)L.c.decay[h];
          a[h] = L.c.decay[h] > 0.0 ? (float)log(L.c.decay[h]) : -1e30f;  // (a finite stand-in for the logarithm of 0)
        }
        DP_TRY(upload_raw(ctx, L.rate, a.data(), a.size() * 4));
        DP_TRY(upload_raw(ctx, L.decay, d.data(), d.size() * 4));
      }
    for (StackLayer &L : s->layers) L.c.decay = nullptr;  // the caller's
    std::vector<HistEntry> entries;
    for (StackLayer &L : s->layers) {
      if (c.input_taps > 1)
        for (int q = 0; q < L.subs(); q++)
          entries.push_back({L.stage[q], L.hist[q], (unsigned long long)c.input_taps * c.width, c.width, c.input_taps});
      if ((L.mamba() || L.is_delta()) && L.c.conv_taps > 1)
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
  for (StackLayer &L : s->layers)
    if (L.owner < 0)
      for (const Mat *t : {&L.proj, &L.o, &L.gateup, &L.down, &L.a2, &L.g2, &L.uq, &L.uk, &L.uv, &L.ukv}) rel(t->buf);
  rel(s->expanded);
  for (RopeTable &t : s->ropes) rel(t.buf);
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
  DP_CHECK(ctx, L.owner < 0, "loadTensor: layer %d uses the tensors of layer %d", layer, L.owner);

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

  auto vec_as = [&](float *dst, int n, auto &&fn) -> dp_status {  // values of a function, element by element
    if (!dst) return dp_fail(ctx, DP_ERR_INVALID, "loadTensor: layer %d has no %s", layer, tensor_name(id));
    DP_TRY(expect(1, n));
    std::vector<float> v;
    for (int i = 0; i < n; i++) {
      const uint32_t bits = (uint32_t)((const uint16_t *)host)[i] << 16;
      float x;
      memcpy(&x, &bits, 4);
      fn(v, x);
    }
    return upload_raw(ctx, dst, v.data(), v.size() * 4);
  };

  const bool att = L.attention(), lig = L.lightning(), del = L.is_delta(), lat = L.latent();
  const int QK = L.delta.qk(), inner = L.inner(), vtaps = L.c.conv_taps;
  dp_status st = DP_OK;
  switch (id) {
    case DP_T_NORM1: st = vec_bf16(L.norm[0], 1, H); break;
    case DP_T_NORM2: st = vec_bf16(L.norm[1], 1, H); break;
    case DP_T_NORM1B: st = vec_bf16(L.post[0], 1, H); break;
    case DP_T_NORM2B: st = vec_bf16(L.post[1], 1, H); break;
    case DP_T_CONV1: st = vec_bf16(L.conv[0], H, taps); break;
    case DP_T_CONV2: st = vec_bf16(L.conv[1], H, taps); break;
    case DP_T_HC1_IN: case DP_T_HC1_OUT: case DP_T_HC1_MIX: case DP_T_HC2_IN: case DP_T_HC2_OUT: case DP_T_HC2_MIX: {
      DP_CHECK(ctx, !s->cfg.post_norm, "loadTensor: layer %d has no %s", layer, tensor_name(id));
      const int q = id >= DP_T_HC2_IN ? 1 : 0, which = id - (q ? DP_T_HC2_IN : DP_T_HC1_IN);
      st = which == 0 ? vec_f32(L.hc_in[q], 1, S) : which == 1 ? vec_f32(L.hc_out[q], 1, S) : vec_f32(L.hc_mix[q], S, S);
      break;
    }
    case DP_T_Q:
      if (lig) st = part(true, L.proj, 2 * inner + L.c.heads * L.c.dim, L.c.heads * L.c.dim, H);
      else if (del) st = part(true, L.proj, 0, QK, H);
      else st = part(att, L.proj, 0, L.q_cols(), H);
      break;
    case DP_T_K:
      if (lig) st = part(true, L.proj, 2 * inner, L.c.heads * L.c.dim, H);
      else if (del) st = part(true, L.proj, QK, QK, H);
      else st = part(att, L.proj, L.q_cols(), L.k_cols(), H);
      break;
    case DP_T_V:
      if (lig) st = part(true, L.proj, inner, inner, H);
      else if (del) st = part(true, L.proj, 2 * QK, inner, H);
      else st = part(att, L.proj, L.q_cols() + L.k_cols(), L.v_cols(), H);
      break;
    case DP_T_GATE_HEADS:
      st = part((att || lat) && L.c.head_gate, L.proj, lat ? L.lat.gate_col() : L.q_cols() + L.k_cols() + L.v_cols(), L.c.heads, H);
      break;
    case DP_T_O: st = part(true, L.o, 0, H, inner); break;
    case DP_T_SSM_IN: st = part(L.mamba(), L.proj, 0, L.proj.N, H); break;
    case DP_T_SSM_CONV: st = vec_f32(L.mamba() ? L.conv_w : nullptr, L.channels(), vtaps); break;
    case DP_T_SSM_CONV_B: st = vec_f32(L.conv_b, 1, L.channels()); break;
    case DP_T_SSM_DT_BIAS: st = vec_f32(L.mamba() ? L.dt_bias : nullptr, 1, L.c.heads); break;
    case DP_T_SSM_A_LOG: st = vec_as(L.mamba() ? L.rate : nullptr, L.c.heads, [](std::vector<float> &v, float x) { v.push_back(-expf(x)); }); break;
    case DP_T_SSM_D: st = vec_f32(L.d, 1, L.c.heads); break;
    case DP_T_SSM_NORM: st = vec_bf16(L.mamba() ? L.mix_norm : nullptr, 1, inner); break;
    case DP_T_GATE: st = part(lig, L.proj, 0, inner, H); break;
    case DP_T_MIX_NORM: st = vec_bf16(lig || del ? L.mix_norm : nullptr, 1, lig ? inner : L.c.vdim); break;
    case DP_T_CONV_Q: st = vec_f32(del ? L.conv_w : nullptr, QK, vtaps); break;
    case DP_T_CONV_K: st = vec_f32(del ? L.conv_w + (size_t)QK * vtaps : nullptr, QK, vtaps); break;
    case DP_T_CONV_V: st = vec_f32(del ? L.conv_w + (size_t)2 * QK * vtaps : nullptr, inner, vtaps); break;
    case DP_T_BETA: st = part(del, L.proj, L.delta.beta_col(), L.c.heads, H); break;
    case DP_T_A1: st = part(del, L.proj, L.delta.a1_col(), L.c.decay_rank, H); break;
    case DP_T_G1: st = part(del, L.proj, L.delta.g1_col(), L.c.gate_rank, H); break;
    case DP_T_A2: st = part(del, L.a2, 0, L.c.heads * L.c.dim, L.c.decay_rank); break;
    case DP_T_G2: st = part(del, L.g2, 0, inner, L.c.gate_rank); break;
    case DP_T_A_LOG:
      st = vec_as(del ? L.rate : nullptr, L.c.heads, [&](std::vector<float> &v, float x) { v.insert(v.end(), (size_t)L.c.dim, expf(x)); });
      break;
    case DP_T_DT_BIAS: st = vec_f32(del ? L.dt_bias : nullptr, 1, L.c.heads * L.c.dim); break;
    case DP_T_DQ: st = part(lat, L.proj, 0, L.c.q_rank, H); break;
    case DP_T_DKV: st = part(lat, L.proj, L.lat.dkv_col(), L.c.kv_rank + L.c.rot_dim, H); break;
    case DP_T_DQ_NORM: st = vec_bf16(L.dq_norm, 1, L.c.q_rank); break;
    case DP_T_DKV_NORM: st = vec_bf16(L.dkv_norm, 1, L.c.kv_rank); break;
    case DP_T_UQ: st = part(lat, L.uq, 0, L.uq.N, L.c.q_rank); break;
    case DP_T_UK:
    case DP_T_UV: {
      const bool is_v = id == DP_T_UV;
      const Mat &w = is_v ? L.uv : L.uk;
      st = part(lat, w, 0, w.N, L.c.kv_rank);
      if (st == DP_OK && L.ukv.buf) {
        st = mat_upload_f16(ctx, L.ukv, is_v ? (int)(L.c.heads * up(L.c.dim, 8)) : 0, host, L.c.heads, is_v ? L.c.vdim : L.c.dim, L.c.kv_rank, &L.up_exact);
        for (StackLayer &o : s->layers)
          if (o.owner == layer) o.up_exact = L.up_exact;
      }
      break;
    }
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
                          single && !s->cfg.post_norm ? m->h : nullptr, rows);
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
    if (s->pending >= 0 && hrow == m->h) {  // a decode row whose last residual sum is still to be done
      p.x = s->x[s->pending]; p.res = s->pending_end; p.res_y = s->y; p.x_out = m->h;
      s->pending = -1;
      return dpk_gemv_bf16(m->ctx, GEMV_SRC_RESIDUAL, GEMV_DST_PLAIN, p);
    }
    return dpk_gemv_bf16(m->ctx, GEMV_SRC_NORM, GEMV_DST_PLAIN, p);
  }
  const int st = a_stride(s, s->cfg.width);
  GroupNorm n;
  n.w = s->final_norm; n.groups = s->cfg.norm_groups; n.eps = s->cfg.eps;
  DP_TRY(dpk_group_norm(m->ctx, hrow, s->cfg.width, n, s->cfg.width, s->a, !s->f32, st, rows));
  return product(m, s->embed, s->a, st, m->logits, rows);
}
