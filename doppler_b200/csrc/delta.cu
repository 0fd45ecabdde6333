// Gated delta rule with one decay per head and key channel, in f32:
//   S <- diag(g) S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q
// q, k (of kv_heads heads) and v through a causal depthwise convolution and silu, q and k then unit vectors per head (q also
// divided by sqrt(dim)), beta = sigmoid(b), g = exp(-exp(A_log) softplus(W_a2 a1 + dt_bias)).
//
// State layout as in ssm.cu: [head][vdim][state_stride], the key channel fastest and padded with zeros to 32 * 2^k; eight
// lanes cover a column with 16-byte pieces (lane s holds channels 4 s + 32 i + {0..3}) and reduce over the channels with
// three shuffles.  A sequence at position 0 starts from zeros whatever its slot held before.
//
// With S already decayed the read-out needs no second pass over the new state: o = S^T q + (k . q) u, so both sums over the
// channels run on the same values and only the one with k is on the path from token to token.  State arithmetic is
// packed two channels at a time (fma.rn.f32x2).
#include "layers.h"
#include "pdl.cuh"

namespace {

constexpr int DL_COLS = 32, DL_LANES = 8, DL_THREADS = DL_COLS * DL_LANES;

__device__ __forceinline__ float dl_silu(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float dl_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float dl_softplus(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float dl_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 x2_pack(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float x2_sum(f32x2 v) {
  float a, b;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
  return a + b;
}
__device__ __forceinline__ f32x2 x2_fma(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 x2_mul(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ void x2_load4(const float *p, f32x2 &a, f32x2 &b) {  // 16-byte aligned
  const ulonglong2 v = *reinterpret_cast<const ulonglong2 *>(p);
  a = v.x; b = v.y;
}
__device__ __forceinline__ void x2_store4(float *p, f32x2 a, f32x2 b) { *reinterpret_cast<ulonglong2 *>(p) = make_ulonglong2(a, b); }

// one token on a column's share of the state: decay, both sums, write.  Returns the read-out (in every lane of the column).
template <int NV>
__device__ __forceinline__ float dl_token(f32x2 (&s)[2 * NV], const float *k, const float *q, const float *g, int sub, float v, float beta, float qk, float k_scale,
                                          float q_scale) {
  f32x2 kk[2 * NV], sk[2] = {0ull, 0ull}, sq[2] = {0ull, 0ull};
#pragma unroll
  for (int i = 0; i < NV; i++) {
    f32x2 g0, g1;
    x2_load4(g + 4 * sub + 32 * i, g0, g1);
    x2_load4(k + 4 * sub + 32 * i, kk[2 * i], kk[2 * i + 1]);
    s[2 * i] = x2_mul(s[2 * i], g0);
    s[2 * i + 1] = x2_mul(s[2 * i + 1], g1);
    sk[0] = x2_fma(s[2 * i], kk[2 * i], sk[0]);
    sk[1] = x2_fma(s[2 * i + 1], kk[2 * i + 1], sk[1]);
  }
  float dk = x2_sum(sk[0]) + x2_sum(sk[1]);
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) dk += __shfl_xor_sync(0xffffffffu, dk, o);
#pragma unroll
  for (int i = 0; i < NV; i++) {
    f32x2 q0, q1;
    x2_load4(q + 4 * sub + 32 * i, q0, q1);
    sq[0] = x2_fma(s[2 * i], q0, sq[0]);
    sq[1] = x2_fma(s[2 * i + 1], q1, sq[1]);
  }
  const float u = beta * fmaf(-k_scale, dk, v);
  const float ku = k_scale * u;
  const f32x2 uu = x2_pack(ku, ku);
#pragma unroll
  for (int i = 0; i < 2 * NV; i++) s[i] = x2_fma(kk[i], uu, s[i]);
  float dq = x2_sum(sq[0]) + x2_sum(sq[1]);
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) dq += __shfl_xor_sync(0xffffffffu, dq, o);
  return q_scale * fmaf(qk, ku, dq);
}

// value of a channel's convolution at row r of a portion, before its silu; r - taps + 1 may reach into the history
__device__ __forceinline__ float dl_conv(const float *proj, int proj_stride, const float *conv, int taps, const float *hist, int CH, int ch, int r, int start_pos) {
  float acc = 0.0f;
  for (int j = 0; j < taps; j++) {
    const int rr = r - (taps - 1) + j, p = start_pos + rr;
    float x = 0.0f;
    if (rr >= 0) x = proj[(size_t)rr * proj_stride + ch];
    else if (p >= 0) x = hist[(size_t)(p % taps) * CH + ch];
    acc = fmaf(conv[(size_t)ch * taps + j], x, acc);
  }
  return acc;
}

// ---- one token per row, rows are sequences: grid (heads, column tiles, rows) ----
// What earlier steps left (state, convolution histories, positions) and the matrices of decay and gate are read before
// griddepcontrol.wait; after it only this token's projections are.
struct DeltaStepSmem {  // offsets in floats; the weight tiles behind them in bytes
  int q, k, v, g, low, red, weights;
  int w_rows_a, w_rows_g, pitch_a, pitch_g;  // staged rows (0: read from global memory), bytes per staged row
  int total;
};

__host__ __device__ inline DeltaStepSmem delta_step_smem(const DeltaShape &sh, int a2_stride, int g2_stride, int limit) {
  DeltaStepSmem m;
  const int NP = sh.state_stride;
  m.q = 0; m.k = NP; m.g = 2 * NP; m.v = 3 * NP; m.low = m.v + DL_COLS;
  m.red = m.low + a2_stride + g2_stride;
  m.weights = (m.red + 16 + 3) / 4 * 4;
  m.pitch_a = a2_stride * 2 + 16; m.pitch_g = g2_stride * 2 + 16;
  m.w_rows_a = sh.dim; m.w_rows_g = DL_COLS;
  m.total = m.weights * 4 + m.w_rows_a * m.pitch_a + m.w_rows_g * m.pitch_g;
  if (m.total > limit) { m.w_rows_a = m.w_rows_g = 0; m.total = m.weights * 4; }
  return m;
}

__device__ __forceinline__ float dl_dot_row(const __nv_bfloat16 *w, const float *x, int pieces, int p0, int step) {
  float acc = 0.0f;
#pragma unroll 4
  for (int i = p0; i < pieces; i += step) {
    const uint4 r = *reinterpret_cast<const uint4 *>(w + 8 * i);
    const float4 a = *reinterpret_cast<const float4 *>(x + 8 * i), b = *reinterpret_cast<const float4 *>(x + 8 * i + 4);
    acc = fmaf(__uint_as_float(r.x << 16), a.x, acc); acc = fmaf(__uint_as_float(r.x & 0xffff0000u), a.y, acc);
    acc = fmaf(__uint_as_float(r.y << 16), a.z, acc); acc = fmaf(__uint_as_float(r.y & 0xffff0000u), a.w, acc);
    acc = fmaf(__uint_as_float(r.z << 16), b.x, acc); acc = fmaf(__uint_as_float(r.z & 0xffff0000u), b.y, acc);
    acc = fmaf(__uint_as_float(r.w << 16), b.z, acc); acc = fmaf(__uint_as_float(r.w & 0xffff0000u), b.w, acc);
  }
  return acc;
}

template <int NV>
__global__ void __launch_bounds__(DL_THREADS) delta_step_kernel(const float *__restrict__ proj, int proj_stride, const DeltaShape sh, const DeltaWeights w,
                                                                const SsmState st, float *__restrict__ out, float *__restrict__ gate,
                                                                const int *__restrict__ pos_arr, const DeltaStepSmem m) {
  constexpr int NP = NV * 32, CHANNELS = 2 * NP + DL_COLS, PER = (CHANNELS + DL_THREADS - 1) / DL_THREADS;
  extern __shared__ __align__(16) float dl_smem[];
  float *sq = dl_smem + m.q, *sk = dl_smem + m.k, *sv = dl_smem + m.v, *sg = dl_smem + m.g, *low_a = dl_smem + m.low, *low_g = low_a + w.a2_stride;
  float *red = dl_smem + m.red;
  unsigned char *s_wa = reinterpret_cast<unsigned char *>(dl_smem + m.weights), *s_wg = s_wa + m.w_rows_a * m.pitch_a;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, p0 = blockIdx.y * DL_COLS, row = blockIdx.z;
  const int D = sh.dim, V = sh.vdim, per = sh.heads / sh.kv_heads, kvh = h / per, CH = sh.channels(), taps = sh.taps, QK = sh.qk(), inner = sh.inner();
  const int cols = min(DL_COLS, V - p0), col = tid / DL_LANES, sub = tid % DL_LANES;
  const int pos = pos_arr[row];
  const float *pr = proj + (size_t)row * proj_stride;
  float *hist = st.hist + (size_t)row * st.hist_seq;
  float *slot = hist + (size_t)(pos % taps) * CH;

  // rows of the decay's and the gate's second matrix
  const __nv_bfloat16 *wa = w.a2 + (size_t)h * D * w.a2_stride, *wg = w.g2 + ((size_t)h * V + p0) * w.g2_stride;
  const int pa = w.a2_stride / 8, pg = w.g2_stride / 8;
  if (m.w_rows_a) {
    for (int i = tid; i < D * pa; i += DL_THREADS)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(s_wa + (i / pa) * m.pitch_a + (i % pa) * 16)), "l"(wa + 8 * (size_t)i) : "memory");
    for (int i = tid; i < cols * pg; i += DL_THREADS)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(s_wg + (i / pg) * m.pitch_g + (i % pg) * 16)), "l"(wg + 8 * (size_t)i) : "memory");
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  float *S = st.s + (size_t)row * st.s_seq + ((size_t)h * V + p0 + col) * NP + 4 * sub;
  f32x2 s[2 * NV];
#pragma unroll
  for (int i = 0; i < NV; i++) {
    if (col < cols && pos > 0) x2_load4(S + 32 * i, s[2 * i], s[2 * i + 1]);
    else s[2 * i] = s[2 * i + 1] = 0ull;
  }
  float acc[PER], last[PER];
  int chan[PER];
#pragma unroll
  for (int j = 0; j < PER; j++) {
    const int i = tid + j * DL_THREADS;
    int ch = -1;
    if (i < 2 * NP) {
      const int n = i < NP ? i : i - NP;
      if (n < D) ch = (i < NP ? 0 : QK) + kvh * D + n;
    } else if (i < 2 * NP + cols) ch = 2 * QK + h * V + p0 + i - 2 * NP;
    chan[j] = ch;
    acc[j] = last[j] = 0.0f;
    if (ch >= 0) {
      const float *cw = w.conv + (size_t)ch * taps;
      last[j] = cw[taps - 1];
      for (int k = taps - 1; k > 0; k--)
        if (pos - k >= 0) acc[j] = fmaf(cw[taps - 1 - k], hist[(size_t)((pos - k) % taps) * CH + ch], acc[j]);
    }
  }
  const bool keep_qk = blockIdx.y == 0 && h == kvh * per;  // one head of the group appends its q and k
  pdl_wait();
  pdl_launch();
  const float beta = dl_sigmoid(pr[sh.beta_col() + h]);
  for (int i = tid; i < w.a2_stride; i += DL_THREADS) low_a[i] = i < sh.decay_rank ? pr[sh.a1_col() + i] : 0.0f;
  for (int i = tid; i < w.g2_stride; i += DL_THREADS) low_g[i] = i < sh.gate_rank ? pr[sh.g1_col() + i] : 0.0f;
#pragma unroll
  for (int j = 0; j < PER; j++) {
    const int i = tid + j * DL_THREADS;
    if (i < CHANNELS) {
      float val = 0.0f;
      if (chan[j] >= 0) {
        const float cur = pr[chan[j]];
        val = dl_silu(fmaf(last[j], cur, acc[j]));
        if (taps > 1 && (i >= 2 * NP || keep_qk)) slot[chan[j]] = cur;
      }
      if (i < NP) sq[i] = val;
      else if (i < 2 * NP) sk[i - NP] = val;
      else sv[i - 2 * NP] = val;
    }
  }
  if (m.w_rows_a) asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  // two threads per key channel: its decay
  for (int c0 = 0; c0 < NP; c0 += DL_THREADS / 2) {
    const int c = c0 + (tid >> 1);
    float d = 0.0f;
    if (c < D) d = dl_dot_row(m.w_rows_a ? reinterpret_cast<const __nv_bfloat16 *>(s_wa + c * m.pitch_a) : wa + (size_t)c * w.a2_stride, low_a, pa, tid & 1, 2);
    d += __shfl_xor_sync(0xffffffffu, d, 1);
    if (c < NP && (tid & 1) == 0) sg[c] = c < D ? expf(-w.rate[h * D + c] * dl_softplus(d + w.bias[h * D + c])) : 0.0f;
  }
  // eight threads per value column: the output gate
  {
    float d = 0.0f;
    if (col < cols) d = dl_dot_row(m.w_rows_a ? reinterpret_cast<const __nv_bfloat16 *>(s_wg + col * m.pitch_g) : wg + (size_t)col * w.g2_stride, low_g, pg, sub, DL_LANES);
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
    if (sub == 0 && col < cols) gate[(size_t)row * inner + h * V + p0 + col] = d;
  }
  if (warp < 3) {  // q.q, k.k, q.k
    const float *a = warp == 1 ? sk : sq, *b = warp == 0 ? sq : sk;
    float d = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; i++) d = fmaf(a[lane + 32 * i], b[lane + 32 * i], d);
    d = dl_warp_sum(d);
    if (lane == 0) red[warp] = d;
  }
  __syncthreads();
  const float q_scale = 1.0f / sqrtf(red[0] + 1e-6f) / sqrtf((float)D), k_scale = 1.0f / sqrtf(red[1] + 1e-6f);
  const float o = dl_token<NV>(s, sk, sq, sg, sub, sv[col], beta, red[2], k_scale, q_scale);
  if (col < cols) {
#pragma unroll
    for (int i = 0; i < NV; i++) x2_store4(S + 32 * i, s[2 * i], s[2 * i + 1]);
    if (sub == 0) out[(size_t)row * inner + h * V + p0 + col] = o;
  }
}

// ---- several tokens of one sequence: everything but the recurrence.  A warp owns 16 rows of a q/k head pair or of a run of
// 32 NJ value channels; the last warps copy the low-rank rows and the write strengths ----
constexpr int DR_ROWS = 16;
template <int NJ>
__global__ void __launch_bounds__(128) delta_rows_kernel(const float *__restrict__ proj, int proj_stride, const DeltaShape sh, const DeltaWeights w, const SsmState st,
                                                         const DeltaRows out, int v_units, int rows, int start_pos, int seq) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31, unit = blockIdx.x * 4 + (threadIdx.x >> 5);
  const int r0 = blockIdx.y * DR_ROWS, r1 = min(r0 + DR_ROWS, rows);
  const int G = sh.kv_heads, D = sh.dim, QK = sh.qk(), CH = sh.channels(), taps = sh.taps, inner = sh.inner();
  const float *hist = st.hist + (size_t)seq * st.hist_seq;
  auto keep = [&](int r, int ch) {  // rows later tokens reach back to
    if (r >= rows - (taps - 1)) st.stage[(size_t)((start_pos + r) % taps) * CH + ch] = proj[(size_t)r * proj_stride + ch];
  };
  if (unit < G) {
    const float q_mul = 1.0f / sqrtf((float)D);
    for (int r = r0; r < r1; r++) {
      float q[NJ], k[NJ], qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
      for (int j = 0; j < NJ; j++) {
        const int d = lane + 32 * j, cq = unit * D + d, ck = QK + cq;
        q[j] = k[j] = 0.0f;
        if (d < D) {
          q[j] = dl_silu(dl_conv(proj, proj_stride, w.conv, taps, hist, CH, cq, r, start_pos));
          k[j] = dl_silu(dl_conv(proj, proj_stride, w.conv, taps, hist, CH, ck, r, start_pos));
          keep(r, cq);
          keep(r, ck);
        }
        qq = fmaf(q[j], q[j], qq);
        kk = fmaf(k[j], k[j], kk);
        qk = fmaf(q[j], k[j], qk);
      }
      qq = dl_warp_sum(qq); kk = dl_warp_sum(kk); qk = dl_warp_sum(qk);
      const float qs = 1.0f / sqrtf(qq + 1e-6f) * q_mul, ks = 1.0f / sqrtf(kk + 1e-6f);
#pragma unroll
      for (int j = 0; j < NJ; j++) {
        const int d = lane + 32 * j;
        if (d < D) {
          out.q[(size_t)r * QK + unit * D + d] = q[j] * qs;
          out.k[(size_t)r * QK + unit * D + d] = k[j] * ks;
        }
      }
      if (lane == 0) out.qk[(size_t)r * G + unit] = qk * qs * ks;
    }
  } else if (unit < G + v_units) {
    for (int r = r0; r < r1; r++)
#pragma unroll
      for (int j = 0; j < NJ; j++) {
        const int e = (unit - G) * 32 * NJ + lane + 32 * j;
        if (e < inner) {
          out.v[(size_t)r * inner + e] = dl_silu(dl_conv(proj, proj_stride, w.conv, taps, hist, CH, 2 * QK + e, r, start_pos));
          keep(r, 2 * QK + e);
        }
      }
  } else if (unit == G + v_units) {
    for (int r = r0; r < r1; r++) {
      const float *pr = proj + (size_t)r * proj_stride;
      for (int i = lane; i < sh.heads; i += 32) out.beta[(size_t)r * sh.heads + i] = dl_sigmoid(pr[sh.beta_col() + i]);
      if (out.a_low)
        for (int i = lane; i < out.a_low_stride; i += 32) out.a_low[(size_t)r * out.a_low_stride + i] = __float2bfloat16_rn(i < sh.decay_rank ? pr[sh.a1_col() + i] : 0.0f);
      if (out.g_low)
        for (int i = lane; i < out.g_low_stride; i += 32) out.g_low[(size_t)r * out.g_low_stride + i] = __float2bfloat16_rn(i < sh.gate_rank ? pr[sh.g1_col() + i] : 0.0f);
    }
  }
}

// ---- the recurrence, token by token: grid (heads, column tiles) ----
constexpr int DS_TB = 16;  // tokens staged at a time
template <int NV>
__global__ void __launch_bounds__(DL_THREADS) delta_scan_kernel(const DeltaShape sh, const SsmState st, const DeltaRows in, float *__restrict__ out, int rows,
                                                                int start_pos, int seq) {
  pdl_launch();
  pdl_wait();
  constexpr int NP = NV * 32, TOK = 3 * NP + DL_COLS + 4;  // floats staged per token: k, q, g, v, beta, q . k
  extern __shared__ __align__(16) float ds_smem[];          // [2][DS_TB][TOK], then o [DS_TB][DL_COLS]
  float *so = ds_smem + 2 * DS_TB * TOK;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, p0 = blockIdx.y * DL_COLS;
  const int D = sh.dim, V = sh.vdim, G = sh.kv_heads, kvh = h / (sh.heads / G), QK = sh.qk(), inner = sh.inner(), HD = sh.heads * D;
  const int cols = min(DL_COLS, V - p0), col = tid / DL_LANES, sub = tid % DL_LANES;
  for (int i = tid; i < 2 * DS_TB * TOK; i += DL_THREADS) ds_smem[i] = 0.0f;  // padded channels and columns stay zero
  __syncthreads();
  const bool vec = (D & 3) == 0 && (V & 3) == 0;
  auto cp = [](float *dst, const float *src, bool wide) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    if (wide) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
  };
  auto stage = [&](int blk) {
    const int r0 = blk * DS_TB, n = min(DS_TB, rows - r0);
    const int unit = vec ? 4 : 1;
    for (int t = warp; t < n; t += DL_THREADS / 32) {
      float *d = ds_smem + ((blk & 1) * DS_TB + t) * TOK;
      const size_t r = (size_t)(r0 + t);
      const float *k = in.k + r * QK + kvh * D, *q = in.q + r * QK + kvh * D, *g = in.g + r * HD + h * D, *v = in.v + r * inner + h * V + p0;
      for (int e = lane * unit; e < D; e += 32 * unit) {
        cp(d + e, k + e, vec);
        cp(d + NP + e, q + e, vec);
        cp(d + 2 * NP + e, g + e, vec);
      }
      for (int e = lane * unit; e < cols; e += 32 * unit) cp(d + 3 * NP + e, v + e, vec);
      if (lane == 0) cp(d + 3 * NP + DL_COLS, in.beta + r * sh.heads + h, false);
      if (lane == 1) cp(d + 3 * NP + DL_COLS + 1, in.qk + r * G + kvh, false);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float *S = st.s + (size_t)seq * st.s_seq + ((size_t)h * V + p0 + col) * NP + 4 * sub;
  f32x2 s[2 * NV];
#pragma unroll
  for (int i = 0; i < NV; i++) {
    if (col < cols && start_pos > 0) x2_load4(S + 32 * i, s[2 * i], s[2 * i + 1]);
    else s[2 * i] = s[2 * i + 1] = 0ull;
  }
  const int blocks = (rows + DS_TB - 1) / DS_TB;
  stage(0);
  for (int blk = 0; blk < blocks; blk++) {
    if (blk + 1 < blocks) {
      stage(blk + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float *src = ds_smem + (blk & 1) * DS_TB * TOK;
    const int r0 = blk * DS_TB, n = min(DS_TB, rows - r0);
#pragma unroll 2
    for (int t = 0; t < n; t++) {
      const float *d = src + t * TOK;
      const float2 bq = *reinterpret_cast<const float2 *>(d + 3 * NP + DL_COLS);
      const float o = dl_token<NV>(s, d, d + NP, d + 2 * NP, sub, d[3 * NP + col], bq.x, bq.y, 1.0f, 1.0f);
      if (sub == 0) so[t * DL_COLS + col] = o;
    }
    __syncthreads();
    for (int i = tid; i < n * DL_COLS; i += DL_THREADS) {
      const int t = i / DL_COLS, c = i - t * DL_COLS;
      if (c < cols) out[(size_t)(r0 + t) * inner + h * V + p0 + c] = so[i];
    }
  }
  if (col < cols)
#pragma unroll
    for (int i = 0; i < NV; i++) x2_store4(S + 32 * i, s[2 * i], s[2 * i + 1]);
}

template <int NV>
dp_status launch_step(dp_ctx *ctx, const float *proj, int proj_stride, const DeltaShape &sh, const DeltaWeights &w, const SsmState &st, float *out, float *gate,
                      int rows, const int *pos) {
  const int limit = 100 * 1024;  // two CTAs per SM
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    DP_CUDA(ctx, cudaFuncSetAttribute(delta_step_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, limit));
    attr.done(ctx->device);
  }
  const DeltaStepSmem m = delta_step_smem(sh, w.a2_stride, w.g2_stride, limit);
  if (m.total > limit) return dp_fail(ctx, DP_ERR_UNSUPPORTED, "delta: low-rank sizes %d and %d exceed shared memory", sh.decay_rank, sh.gate_rank);
  DP_LAUNCH(ctx, delta_step_kernel<NV>, dim3(sh.heads, (sh.vdim + DL_COLS - 1) / DL_COLS, rows), DL_THREADS, (size_t)m.total, proj, proj_stride, sh, w, st, out, gate,
            pos, m);
  return DP_OK;
}

template <int NV>
dp_status launch_scan(dp_ctx *ctx, const DeltaShape &sh, const SsmState &st, const DeltaRows &r, float *out, int rows, const RowMap &map) {
  const size_t smem = (size_t)(2 * DS_TB * (3 * NV * 32 + DL_COLS + 4) + DS_TB * DL_COLS) * 4;
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    DP_CUDA(ctx, cudaFuncSetAttribute(delta_scan_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr.done(ctx->device);
  }
  DP_LAUNCH(ctx, delta_scan_kernel<NV>, dim3(sh.heads, (sh.vdim + DL_COLS - 1) / DL_COLS), DL_THREADS, smem, sh, st, r, out, rows, map.start_pos, map.seq);
  return DP_OK;
}

template <int NJ>
dp_status launch_rows(dp_ctx *ctx, const float *proj, int proj_stride, const DeltaShape &sh, const DeltaWeights &w, const SsmState &st, const DeltaRows &r, int rows,
                      const RowMap &map) {
  const int v_units = (sh.inner() + 32 * NJ - 1) / (32 * NJ), units = sh.kv_heads + v_units + 1;
  DP_LAUNCH(ctx, delta_rows_kernel<NJ>, dim3((units + 3) / 4, (rows + DR_ROWS - 1) / DR_ROWS), 128, 0, proj, proj_stride, sh, w, st, r, v_units, rows, map.start_pos,
            map.seq);
  return DP_OK;
}

}  // namespace

#define DP_BY_STRIDE(fn, ...)                       \
  switch (sh.state_stride / 32) {                   \
    case 1: return fn<1>(__VA_ARGS__);              \
    case 2: return fn<2>(__VA_ARGS__);              \
    case 4: return fn<4>(__VA_ARGS__);              \
    case 8: return fn<8>(__VA_ARGS__);              \
    case 16: return fn<16>(__VA_ARGS__);            \
  }                                                 \
  return dp_fail(ctx, DP_ERR_UNSUPPORTED, "delta: key size %d", sh.dim)

dp_status dpk_delta_step(dp_ctx *ctx, const float *proj, int proj_stride, const DeltaShape &sh, const DeltaWeights &w, const SsmState &st, float *out,
                         float *gate, int rows, const int *pos) {
  DP_BY_STRIDE(launch_step, ctx, proj, proj_stride, sh, w, st, out, gate, rows, pos);
}
dp_status dpk_delta_rows(dp_ctx *ctx, const float *proj, int proj_stride, const DeltaShape &sh, const DeltaWeights &w, const SsmState &st, const DeltaRows &r,
                         int rows, const RowMap &map) {
  DP_BY_STRIDE(launch_rows, ctx, proj, proj_stride, sh, w, st, r, rows, map);
}
dp_status dpk_delta_scan(dp_ctx *ctx, const DeltaShape &sh, const SsmState &st, const DeltaRows &r, float *out, int rows, const RowMap &map) {
  DP_BY_STRIDE(launch_scan, ctx, sh, st, r, out, rows, map);
}
