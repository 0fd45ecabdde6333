// Gated delta rule with one decay per head and key channel, in f32:
//   S <- diag(g) S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q
// q, k (of kv_heads heads) and v through a causal depthwise convolution and silu, q and k then unit vectors per head (q also
// divided by sqrt(dim)), beta = sigmoid(b), g = exp(-exp(A_log) softplus(W_a2 a1 + dt_bias)).
//
// State layout as in ssm.cu: [head][vdim][state_stride], the key channel fastest and padded with zeros to 32 * 2^k.  A
// sequence at position 0 starts from zeros whatever its slot held before.  State arithmetic is packed two channels at a
// time (fma.rn.f32x2).
//
// A decode step has eight lanes cover a column (lane s holds channels 4 s + 32 i + {0..3}).  With S already decayed the
// read-out needs no second pass over the new state: o = S^T q + (k . q) u.
//
// A portion takes four tokens at a time.  With S the state before them and P(s, t) the product of the decays of tokens
// s + 1 .. t per channel (products only, nothing is ever divided by a decay):
//   u_t = beta_t (v_t - S^T (P(-1, t) k_t) - sum_{s < t} (k_t . P(s, t) k_s) u_s)
//   o_t = S^T (P(-1, t) q_t) + sum_{s <= t} (q_t . P(s, t) k_s) u_s
//   S'  = P(-1, 3) S + sum_s (P(s, 3) k_s) u_s^T
// so the sums over the channels of four tokens are reduced across lanes together and the chain from token to token is a
// handful of scalars.  What does not depend on the state (the vectors in brackets and the scalars) is prepared for all
// heads and blocks at once.
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
  int q, k, v, g, low, weights;
  int w_rows_a, w_rows_g, pitch_a, pitch_g;  // staged rows (0: read from global memory), bytes per staged row
  int total;
};

__host__ __device__ inline DeltaStepSmem delta_step_smem(const DeltaShape &sh, int a2_stride, int g2_stride, int limit, bool staged) {
  DeltaStepSmem m;
  const int NP = sh.state_stride;
  m.q = 0; m.k = NP; m.g = 2 * NP; m.v = 3 * NP; m.low = m.v + DL_COLS;
  m.weights = m.low + a2_stride + g2_stride;  // (a multiple of four)
  m.pitch_a = a2_stride * 2 + 16; m.pitch_g = g2_stride * 2 + 16;
  m.w_rows_a = sh.dim; m.w_rows_g = DL_COLS;
  m.total = m.weights * 4 + m.w_rows_a * m.pitch_a + m.w_rows_g * m.pitch_g;
  if (!staged || m.total > limit) { m.w_rows_a = m.w_rows_g = 0; m.total = m.weights * 4; }
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

// product of one 16-byte piece of a row with eight values
__device__ __forceinline__ float dl_piece(const uint4 &r, const float (&x)[8]) {
  float acc = __uint_as_float(r.x << 16) * x[0];
  acc = fmaf(__uint_as_float(r.x & 0xffff0000u), x[1], acc);
  acc = fmaf(__uint_as_float(r.y << 16), x[2], acc); acc = fmaf(__uint_as_float(r.y & 0xffff0000u), x[3], acc);
  acc = fmaf(__uint_as_float(r.z << 16), x[4], acc); acc = fmaf(__uint_as_float(r.z & 0xffff0000u), x[5], acc);
  acc = fmaf(__uint_as_float(r.w << 16), x[6], acc); acc = fmaf(__uint_as_float(r.w & 0xffff0000u), x[7], acc);
  return acc;
}
// sums over sixteen lanes of N values each (N a power of two up to sixteen): the lane ends up with the sum of value (lane & 15) / (16 / N)
template <int N> __device__ __forceinline__ float dl_sum_scatter16(float (&v)[N], int lane) {
  int n = N;
#pragma unroll
  for (int o = 8; o > 0; o >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool upper = lane & o;
#pragma unroll
      for (int i = 0; i < (N > 1 ? N / 2 : 1); i++)
        if (i < n) {
          const float send = upper ? v[i] : v[i + n], keep = upper ? v[i + n] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
    }
  }
  return v[0];
}

// SMALL: low-rank sizes up to 128.  The matrices' rows are then fetched straight into registers, sixteen lanes to a row.
template <int NV, bool SMALL>
__global__ void __launch_bounds__(DL_THREADS) delta_step_kernel(const float *__restrict__ proj, int proj_stride, const DeltaShape sh, const DeltaWeights w,
                                                                const SsmState st, float *__restrict__ out, float *__restrict__ gate,
                                                                const int *__restrict__ pos_arr, const DeltaStepSmem m) {
  constexpr int NP = NV * 32, CHANNELS = 2 * NP + DL_COLS, PER = (CHANNELS + DL_THREADS - 1) / DL_THREADS;
  extern __shared__ __align__(16) float dl_smem[];
  float *sq = dl_smem + m.q, *sk = dl_smem + m.k, *sv = dl_smem + m.v, *sg = dl_smem + m.g, *low_a = dl_smem + m.low, *low_g = low_a + w.a2_stride;
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
  constexpr int IT = SMALL ? NP / 16 : 1, GT = 2;  // rows per half-warp: key channels, value columns
  const int half = lane >> 4, piece = lane & 15;
  uint4 ra[IT], rg[GT];
  if constexpr (SMALL) {
#pragma unroll
    for (int i = 0; i < IT; i++) {
      const int c = warp * (NP / 8) + 2 * i + half;
      ra[i] = c < D && piece < pa ? __ldg(reinterpret_cast<const uint4 *>(wa + (size_t)c * w.a2_stride) + piece) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int i = 0; i < GT; i++) {
      const int c = warp * 4 + 2 * i + half;
      rg[i] = c < cols && piece < pg ? __ldg(reinterpret_cast<const uint4 *>(wg + (size_t)c * w.g2_stride) + piece) : make_uint4(0, 0, 0, 0);
    }
  } else if (m.w_rows_a) {
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
  // the decay this lane will finish (SMALL): its constants
  const int my_c = warp * (NP / 8) + 2 * (piece / (16 / IT)) + half;
  const float rate = SMALL && my_c < D ? w.rate[h * D + my_c] : 0.0f, bias = SMALL && my_c < D ? w.bias[h * D + my_c] : 0.0f;
  const bool keep_qk = blockIdx.y == 0 && h == kvh * per;  // one head of the group appends its q and k
  pdl_wait();
  pdl_launch();
  const float beta = dl_sigmoid(pr[sh.beta_col() + h]);
  float xa[8], xg[8], cur[PER];
  if constexpr (SMALL) {
#pragma unroll
    for (int j = 0; j < 8; j++) {
      const int i = piece * 8 + j;
      xa[j] = i < sh.decay_rank ? pr[sh.a1_col() + i] : 0.0f;
      xg[j] = i < sh.gate_rank ? pr[sh.g1_col() + i] : 0.0f;
    }
  } else {
    for (int i = tid; i < w.a2_stride; i += DL_THREADS) low_a[i] = i < sh.decay_rank ? pr[sh.a1_col() + i] : 0.0f;
    for (int i = tid; i < w.g2_stride; i += DL_THREADS) low_g[i] = i < sh.gate_rank ? pr[sh.g1_col() + i] : 0.0f;
  }
#pragma unroll
  for (int j = 0; j < PER; j++) cur[j] = chan[j] >= 0 ? pr[chan[j]] : 0.0f;
#pragma unroll
  for (int j = 0; j < PER; j++) {
    const int i = tid + j * DL_THREADS;
    if (i < CHANNELS) {
      float val = 0.0f;
      if (chan[j] >= 0) {
        val = dl_silu(fmaf(last[j], cur[j], acc[j]));
        if (taps > 1 && (i >= 2 * NP || keep_qk)) slot[chan[j]] = cur[j];
      }
      if (i < NP) sq[i] = val;
      else if (i < 2 * NP) sk[i - NP] = val;
      else sv[i - 2 * NP] = val;
    }
  }
  if constexpr (SMALL) {
    float va[IT], vg[GT];
#pragma unroll
    for (int i = 0; i < IT; i++) va[i] = dl_piece(ra[i], xa);
#pragma unroll
    for (int i = 0; i < GT; i++) vg[i] = dl_piece(rg[i], xg);
    const float a = dl_sum_scatter16<IT>(va, lane), g = dl_sum_scatter16<GT>(vg, lane);
    if (piece % (16 / IT) == 0) sg[my_c] = my_c < D ? expf(-rate * dl_softplus(a + bias)) : 0.0f;
    const int gc = warp * 4 + 2 * (piece / (16 / GT)) + half;
    if (piece % (16 / GT) == 0 && gc < cols) gate[(size_t)row * inner + h * V + p0 + gc] = g;
    __syncthreads();
  } else {
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
    float d = 0.0f;
    if (col < cols) d = dl_dot_row(m.w_rows_a ? reinterpret_cast<const __nv_bfloat16 *>(s_wg + col * m.pitch_g) : wg + (size_t)col * w.g2_stride, low_g, pg, sub, DL_LANES);
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
    if (sub == 0 && col < cols) gate[(size_t)row * inner + h * V + p0 + col] = d;
    __syncthreads();
  }
  // q.q, k.k, q.k, by every warp for itself
  float qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const float a = sq[lane + 32 * i], b = sk[lane + 32 * i];
    qq = fmaf(a, a, qq); kk = fmaf(b, b, kk); qk = fmaf(a, b, qk);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    qq += __shfl_xor_sync(0xffffffffu, qq, o);
    kk += __shfl_xor_sync(0xffffffffu, kk, o);
    qk += __shfl_xor_sync(0xffffffffu, qk, o);
  }
  const float q_scale = 1.0f / sqrtf(qq + 1e-6f) / sqrtf((float)D), k_scale = 1.0f / sqrtf(kk + 1e-6f);
  const float o = dl_token<NV>(s, sk, sq, sg, sub, sv[col], beta, qk, k_scale, q_scale);
  if (col < cols) {
#pragma unroll
    for (int i = 0; i < NV; i++) x2_store4(S + 32 * i, s[2 * i], s[2 * i + 1]);
    if (sub == 0) out[(size_t)row * inner + h * V + p0 + col] = o;
  }
}

// ---- several tokens of one sequence: convolutions, unit norms, write strengths ----
constexpr int DR_ROWS = 16;

// write strengths and low-rank rows [r0, r1)
__device__ __forceinline__ void dl_aux_rows(const float *proj, int proj_stride, const DeltaShape &sh, const DeltaRows &out, int lane, int r0, int r1) {
  for (int r = r0; r < r1; r++) {
    const float *pr = proj + (size_t)r * proj_stride;
    for (int i = lane; i < sh.heads; i += 32) out.beta[(size_t)r * sh.heads + i] = dl_sigmoid(pr[sh.beta_col() + i]);
    if (out.a_low)
#pragma unroll 4
      for (int i = lane; i < out.a_low_stride; i += 32) out.a_low[(size_t)r * out.a_low_stride + i] = __float2bfloat16_rn(i < sh.decay_rank ? pr[sh.a1_col() + i] : 0.0f);
    if (out.g_low)
#pragma unroll 4
      for (int i = lane; i < out.g_low_stride; i += 32) out.g_low[(size_t)r * out.g_low_stride + i] = __float2bfloat16_rn(i < sh.gate_rank ? pr[sh.g1_col() + i] : 0.0f);
  }
}
constexpr int DR_AUX = 4;  // warps that share these rows of a block

// Any sizes.  A warp owns 16 rows of a q/k head pair or of a run of 32 NJ value channels.
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
      float q[NJ], k[NJ], qq = 0.0f, kk = 0.0f;
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
      }
      const float qs = 1.0f / sqrtf(dl_warp_sum(qq) + 1e-6f) * q_mul, ks = 1.0f / sqrtf(dl_warp_sum(kk) + 1e-6f);
#pragma unroll
      for (int j = 0; j < NJ; j++) {
        const int d = lane + 32 * j;
        if (d < D) {
          out.q[(size_t)r * QK + unit * D + d] = q[j] * qs;
          out.k[(size_t)r * QK + unit * D + d] = k[j] * ks;
        }
      }
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
  } else if (unit < G + v_units + DR_AUX) {
    const int step = DR_ROWS / DR_AUX, a0 = r0 + (unit - G - v_units) * step;
    dl_aux_rows(proj, proj_stride, sh, out, lane, a0, min(a0 + step, r1));
  }
}

// Up to four taps, sizes and strides that are multiples of four: a lane owns four neighbouring channels (times JV), the
// rows a token reaches back to stay in registers, and four rows are fetched at a time.  FAST: the approximate exponential and
// quotient (the bf16 mode, in which these activations need no more than sixteen bits).
template <int TAPS, bool FAST>
struct ConvWindow {
  static __device__ __forceinline__ float silu(float v) { return FAST ? __fdividef(v, 1.0f + __expf(-v)) : dl_silu(v); }
  float w[4][TAPS];
  float4 win[TAPS];  // the last TAPS rows, newest at the end
  __device__ __forceinline__ void init(const float *conv, const float *proj, int proj_stride, const float *hist, int CH, int ch, int r0, int start_pos) {
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
      for (int k = 0; k < TAPS; k++) w[i][k] = conv[(size_t)(ch + i) * TAPS + k];
#pragma unroll
    for (int k = 0; k + 1 < TAPS; k++) {
      const int r = r0 - (TAPS - 1) + k, p = start_pos + r;
      if (r >= 0) win[k + 1] = *reinterpret_cast<const float4 *>(proj + (size_t)r * proj_stride + ch);
      else if (p >= 0) win[k + 1] = *reinterpret_cast<const float4 *>(hist + (size_t)(p % TAPS) * CH + ch);
      else win[k + 1] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
  }
  __device__ __forceinline__ float4 step(const float4 &x) {  // the row's convolution after silu
#pragma unroll
    for (int k = 0; k + 1 < TAPS; k++) win[k] = win[k + 1];
    win[TAPS - 1] = x;
    float4 o = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int k = 0; k < TAPS; k++) {
      o.x = fmaf(w[0][k], win[k].x, o.x); o.y = fmaf(w[1][k], win[k].y, o.y);
      o.z = fmaf(w[2][k], win[k].z, o.z); o.w = fmaf(w[3][k], win[k].w, o.w);
    }
    return make_float4(silu(o.x), silu(o.y), silu(o.z), silu(o.w));
  }
};

template <int JV, int TAPS, bool FAST>
__global__ void __launch_bounds__(128) delta_rows4_kernel(const float *__restrict__ proj, int proj_stride, const DeltaShape sh, const DeltaWeights w, const SsmState st,
                                                          const DeltaRows out, int v_units, int rows, int start_pos, int seq) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31, unit = blockIdx.x * 4 + (threadIdx.x >> 5);
  const int r0 = blockIdx.y * DR_ROWS, r1 = min(r0 + DR_ROWS, rows);
  const int G = sh.kv_heads, D = sh.dim, QK = sh.qk(), CH = sh.channels(), inner = sh.inner();
  const float *hist = st.hist + (size_t)seq * st.hist_seq;
  constexpr int BATCH = 4;
  auto keep = [&](int r, int ch, const float4 &x) {
    if (TAPS > 1 && r >= rows - (TAPS - 1)) *reinterpret_cast<float4 *>(st.stage + (size_t)((start_pos + r) % TAPS) * CH + ch) = x;
  };
  if (unit < G) {
    const float q_mul = 1.0f / sqrtf((float)D);
    ConvWindow<TAPS, FAST> cq[JV], ck[JV];
#pragma unroll
    for (int j = 0; j < JV; j++) {
      const int d = 4 * lane + 128 * j;
      if (d < D) {
        cq[j].init(w.conv, proj, proj_stride, hist, CH, unit * D + d, r0, start_pos);
        ck[j].init(w.conv, proj, proj_stride, hist, CH, QK + unit * D + d, r0, start_pos);
      }
    }
    for (int rb = r0; rb < r1; rb += BATCH) {
      float4 xq[BATCH][JV], xk[BATCH][JV];
#pragma unroll
      for (int b = 0; b < BATCH; b++)
#pragma unroll
        for (int j = 0; j < JV; j++) {
          const int d = 4 * lane + 128 * j;
          if (d < D && rb + b < r1) {
            xq[b][j] = *reinterpret_cast<const float4 *>(proj + (size_t)(rb + b) * proj_stride + unit * D + d);
            xk[b][j] = *reinterpret_cast<const float4 *>(proj + (size_t)(rb + b) * proj_stride + QK + unit * D + d);
          }
        }
#pragma unroll
      for (int b = 0; b < BATCH; b++) {
        const int r = rb + b;
        if (r >= r1) break;  // warp-uniform
        float qq = 0.0f, kk = 0.0f;
        float4 q[JV], k[JV];
#pragma unroll
        for (int j = 0; j < JV; j++) {
          const int d = 4 * lane + 128 * j;
          q[j] = k[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
          if (d < D) {
            q[j] = cq[j].step(xq[b][j]);
            k[j] = ck[j].step(xk[b][j]);
            keep(r, unit * D + d, xq[b][j]);
            keep(r, QK + unit * D + d, xk[b][j]);
          }
          qq = fmaf(q[j].x, q[j].x, fmaf(q[j].y, q[j].y, fmaf(q[j].z, q[j].z, fmaf(q[j].w, q[j].w, qq))));
          kk = fmaf(k[j].x, k[j].x, fmaf(k[j].y, k[j].y, fmaf(k[j].z, k[j].z, fmaf(k[j].w, k[j].w, kk))));
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
          qq += __shfl_xor_sync(0xffffffffu, qq, o);
          kk += __shfl_xor_sync(0xffffffffu, kk, o);
        }
        const float qs = 1.0f / sqrtf(qq + 1e-6f) * q_mul, ks = 1.0f / sqrtf(kk + 1e-6f);
#pragma unroll
        for (int j = 0; j < JV; j++) {
          const int d = 4 * lane + 128 * j;
          if (d < D) {
            *reinterpret_cast<float4 *>(out.q + (size_t)r * QK + unit * D + d) = make_float4(q[j].x * qs, q[j].y * qs, q[j].z * qs, q[j].w * qs);
            *reinterpret_cast<float4 *>(out.k + (size_t)r * QK + unit * D + d) = make_float4(k[j].x * ks, k[j].y * ks, k[j].z * ks, k[j].w * ks);
          }
        }
      }
    }
  } else if (unit < G + v_units) {
    const int e = (unit - G) * 128 + 4 * lane;
    if (e >= inner) return;
    ConvWindow<TAPS, FAST> cv;
    cv.init(w.conv, proj, proj_stride, hist, CH, 2 * QK + e, r0, start_pos);
    for (int rb = r0; rb < r1; rb += BATCH) {
      float4 x[BATCH];
#pragma unroll
      for (int b = 0; b < BATCH; b++)
        if (rb + b < r1) x[b] = *reinterpret_cast<const float4 *>(proj + (size_t)(rb + b) * proj_stride + 2 * QK + e);
#pragma unroll
      for (int b = 0; b < BATCH; b++)
        if (rb + b < r1) {
          *reinterpret_cast<float4 *>(out.v + (size_t)(rb + b) * inner + e) = cv.step(x[b]);
          keep(rb + b, 2 * QK + e, x[b]);
        }
    }
  } else if (unit < G + v_units + DR_AUX) {
    const int step = DR_ROWS / DR_AUX, a0 = r0 + (unit - G - v_units) * step;
    dl_aux_rows(proj, proj_stride, sh, out, lane, a0, min(a0 + step, r1));
  }
}

// ---- what a block of four tokens brings, without the state: one warp per (block, head) ----
// A record: k and q decayed since the block's start, k decayed until its end (4 x NP each), the block's decay (NP), then
// scalars: [k_1.k_0, k_2.k_0, k_2.k_1, k_3.k_0 | k_3.k_1, k_3.k_2, 0, 0 | beta_0..3 | q_t.k_s as rows t of four], decayed.
constexpr int DB_T = 4, DB_SCALARS = 32;
__host__ __device__ constexpr int db_record(int np) { return (3 * DB_T + 1) * np + DB_SCALARS; }

template <int NP>
__global__ void __launch_bounds__(128) delta_block_kernel(const DeltaShape sh, const DeltaRows in, int rows) {
  pdl_launch();
  pdl_wait();
  constexpr int JB = NP >= 128 ? NP / 128 : 1;
  const int lane = threadIdx.x & 31, unit = blockIdx.x * 4 + (threadIdx.x >> 5);
  const int H = sh.heads, D = sh.dim, QK = sh.qk(), HD = H * D, blocks = (rows + DB_T - 1) / DB_T;
  if (unit >= blocks * H) return;
  const int blk = unit / H, h = unit - blk * H, kvh = h / (H / sh.kv_heads), r0 = blk * DB_T;
  const bool vec = (D & 3) == 0;
  float4 k[DB_T][JB], q[DB_T][JB], g[DB_T][JB];
  auto load = [&](const float *p, int d, bool ok, float fill) {
    float4 v = make_float4(fill, fill, fill, fill);
    if (!ok || d >= D) return v;
    if (vec) return *reinterpret_cast<const float4 *>(p + d);
    v.x = p[d];
    if (d + 1 < D) v.y = p[d + 1];
    if (d + 2 < D) v.z = p[d + 2];
    if (d + 3 < D) v.w = p[d + 3];
    return v;
  };
#pragma unroll
  for (int t = 0; t < DB_T; t++)
#pragma unroll
    for (int j = 0; j < JB; j++) {
      const int d = 4 * lane + 128 * j;
      const bool ok = r0 + t < rows;
      const size_t r = (size_t)(r0 + t);
      k[t][j] = load(in.k + r * QK + kvh * D, d, ok, 0.0f);
      q[t][j] = load(in.q + r * QK + kvh * D, d, ok, 0.0f);
      g[t][j] = load(in.g + r * HD + h * D, d, ok, 1.0f);
    }
  const float beta = lane < DB_T && r0 + lane < rows ? in.beta[(size_t)(r0 + lane) * H + h] : 0.0f;
  float *rec = in.records + (size_t)unit * db_record(NP);
  auto mul = [](float4 &a, const float4 &b) { a.x *= b.x; a.y *= b.y; a.z *= b.z; a.w *= b.w; };
  auto dot = [](const float4 &a, const float4 &b, float c) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, c)))); };
  auto put = [&](int slot, int j, const float4 &v) {
    const int d = 4 * lane + 128 * j;
    if (d < NP) *reinterpret_cast<float4 *>(rec + slot * NP + d) = v;
  };
  // decayed since the start
  float4 c[JB];
#pragma unroll
  for (int t = 0; t < DB_T; t++)
#pragma unroll
    for (int j = 0; j < JB; j++) {
      if (t == 0) c[j] = g[0][j];
      else mul(c[j], g[t][j]);
      float4 a = k[t][j], b = q[t][j];
      mul(a, c[j]);
      mul(b, c[j]);
      put(t, j, a);
      put(DB_T + t, j, b);
      if (t == DB_T - 1) put(3 * DB_T, j, c[j]);
    }
  // decayed from each token on, and the scalars between tokens
  float sum[16];  // 0..5: k.k pairs in record order, 6 + 3 s - s (s - 1) / 2 ... : q_t . k_s for t >= s, s by s
  int n = 6;
#pragma unroll
  for (int s = 0; s < DB_T; s++) {
    float d0 = 0.0f;
#pragma unroll
    for (int j = 0; j < JB; j++) d0 = dot(k[s][j], q[s][j], d0);
    sum[n++] = d0;
#pragma unroll
    for (int t = s + 1; t < DB_T; t++) {
      float kk = 0.0f, kq = 0.0f;
#pragma unroll
      for (int j = 0; j < JB; j++) {
        mul(k[s][j], g[t][j]);
        kk = dot(k[s][j], k[t][j], kk);
        kq = dot(k[s][j], q[t][j], kq);
      }
      sum[t == 1 ? 0 : t == 2 ? 1 + s : 3 + s] = kk;
      sum[n++] = kq;
    }
#pragma unroll
    for (int j = 0; j < JB; j++) put(2 * DB_T + s, j, k[s][j]);
  }
#pragma unroll
  for (int i = 0; i < 16; i++) sum[i] = dl_warp_sum(sum[i]);
  float out = 0.0f;  // lane i writes scalar i
#pragma unroll
  for (int i = 0; i < 6; i++)
    if (lane == i) out = sum[i];
  n = 6;
#pragma unroll
  for (int s = 0; s < DB_T; s++)
#pragma unroll
    for (int t = s; t < DB_T; t++) {
      if (lane == 12 + 4 * t + s) out = sum[n];
      n++;
    }
  const float b = __shfl_sync(0xffffffffu, beta, lane & 3);
  if (lane >= 8 && lane < 12) out = b;
  rec[(3 * DB_T + 1) * NP + lane] = out;
}

// ---- the recurrence: grid (heads, column tiles), a warp per eight columns ----
// LN lanes share LN / 4 columns, a lane holds NP / LN channels of each (4 l + 4 LN i + {0..3}).  The sums of a block (columns x
// tokens x {k, q}) are reduced and scattered at once, half of them handed over in every step: lane 4 c + t of the warp ends up
// with both sums of column c and token t.  Every lane numbers columns and tokens relative to its own (exclusive or), so that
// what it keeps always has the lower numbers and no value is ever selected by lane.  What paces the kernel is shared memory
// (the vectors' way into registers, the exchange of the sums) and the instructions around the multiplications, so a warp
// takes many columns rather than few (128 channels, 1024 tokens: 4 columns 219 us, 8 columns 174 us).
constexpr int DS_COLS = 32, DS_WARPS = 4, DS_THREADS = DS_WARPS * 32, DS_STAGES = 4;
template <int NP, int LN>
__global__ void __launch_bounds__(DS_THREADS) delta_scan_kernel(const DeltaShape sh, const SsmState st, const DeltaRows in, float *__restrict__ out, int rows,
                                                                int start_pos, int seq) {
  pdl_launch();
  pdl_wait();
  constexpr int R4 = NP / LN / 4, C = LN / 4, REC = db_record(NP), PIECES = REC / 4;
  extern __shared__ __align__(16) float ds_smem[];  // [DS_STAGES][REC]
  __shared__ float sv[DS_STAGES][DB_T][DS_COLS];
  __shared__ __align__(16) f32x2 su[DS_WARPS][8][DB_T];  // (u, u)
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, li = lane & (LN - 1), grp = lane / LN;
  const int V = sh.vdim, inner = sh.inner(), H = sh.heads;
  const int c0 = blockIdx.y * DS_COLS + warp * 8;                     // the warp's first column
  const int my_t = lane & 3, my_col = c0 + (lane >> 2), first = lane & ~3;  // what this lane finishes
  auto col_of = [&](int c) { return grp * C + (c ^ (li >> 2)); };          // column of local number c within the warp
  const int blocks = (rows + DB_T - 1) / DB_T;
  const float *src = in.records + (size_t)h * REC + 4 * tid;  // this thread's pieces of the next record to fetch
  const uint32_t dst0 = (uint32_t)__cvta_generic_to_shared(ds_smem) + 16 * tid;
  const bool v_ok = (int)blockIdx.y * DS_COLS + lane < V;
  const float *v_src = in.v + (size_t)(tid >> 5) * inner + (size_t)h * V + blockIdx.y * DS_COLS + lane;
  auto stage = [&](int blk, int slot) {
    if (blk < blocks) {
#pragma unroll
      for (int k = 0; k < (PIECES + DS_THREADS - 1) / DS_THREADS; k++)
        if (tid + k * DS_THREADS < PIECES)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst0 + slot * (REC * 4) + k * (DS_THREADS * 16)), "l"(src + k * (DS_THREADS * 4)) : "memory");
      src += (size_t)H * REC;
      if (tid < DB_T * DS_COLS) {  // the block's values, zeros past the rows and columns
        const bool ok = v_ok && blk * DB_T + (tid >> 5) < rows;
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(&sv[slot][tid >> 5][lane])), "l"(ok ? v_src : in.v),
                     "r"(ok ? 4 : 0) : "memory");
        v_src += (size_t)DB_T * inner;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  f32x2 s[C][2 * R4];
  float *S = st.s + (size_t)seq * st.s_seq + ((size_t)h * V + c0) * NP + 4 * li;
#pragma unroll
  for (int c = 0; c < C; c++)
#pragma unroll
    for (int i = 0; i < R4; i++) {
      if (c0 + col_of(c) < V && start_pos > 0) x2_load4(S + (size_t)col_of(c) * NP + 4 * LN * i, s[c][2 * i], s[c][2 * i + 1]);
      else s[c][2 * i] = s[c][2 * i + 1] = 0ull;
    }
  const size_t step = (size_t)DB_T * inner;
  float *o_ptr = out + (size_t)my_t * inner + (size_t)h * V + my_col;
  int left = my_col < V ? rows - my_t : 0;  // rows this lane still writes from its token on
#pragma unroll
  for (int i = 0; i < DS_STAGES - 1; i++) stage(i, i);
  int slot = 0;
  for (int blk = 0; blk < blocks; blk++) {
    asm volatile("cp.async.wait_group %0;" ::"n"(DS_STAGES - 2) : "memory");
    __syncthreads();  // this record is there, and every warp is done with the one before it
    stage(blk + DS_STAGES - 1, slot == 0 ? DS_STAGES - 1 : slot - 1);
    const float *rec = ds_smem + slot * REC, *vec = rec + 4 * li, *sc = rec + (3 * DB_T + 1) * NP;
    // what does not wait for the sums
    const float v = sv[slot][my_t][warp * 8 + (lane >> 2)];
    slot = slot == DS_STAGES - 1 ? 0 : slot + 1;
    const float4 a0 = *reinterpret_cast<const float4 *>(sc), be = *reinterpret_cast<const float4 *>(sc + 8);
    const float2 a1 = *reinterpret_cast<const float2 *>(sc + 4);
    const float4 b = *reinterpret_cast<const float4 *>(sc + 12 + 4 * my_t);
    float val[C * 2 * DB_T];
#pragma unroll
    for (int t = 0; t < DB_T; t++)
#pragma unroll
      for (int kq = 0; kq < 2; kq++) {
        const float *p = vec + (kq * DB_T + (t ^ my_t)) * NP;
        f32x2 x[2 * R4], acc[C];
#pragma unroll
        for (int i = 0; i < R4; i++) x2_load4(p + 4 * LN * i, x[2 * i], x[2 * i + 1]);
#pragma unroll
        for (int c = 0; c < C; c++) {
          acc[c] = x2_mul(s[c][0], x[0]);
#pragma unroll
          for (int i = 1; i < 2 * R4; i++) acc[c] = x2_fma(s[c][i], x[i], acc[c]);
        }
#pragma unroll
        for (int c = 0; c < C; c++) val[(c * DB_T + t) * 2 + kq] = x2_sum(acc[c]);
      }
    constexpr bool EARLY = R4 == 1;  // (registers)
    f32x2 kx[EARLY ? DB_T : 1][2 * R4];
    if constexpr (EARLY) {
#pragma unroll
      for (int t = 0; t < DB_T; t++) x2_load4(vec + (2 * DB_T + t) * NP, kx[t][0], kx[t][1]);
    }
    {
      f32x2 g[2 * R4];
#pragma unroll
      for (int i = 0; i < R4; i++) x2_load4(vec + 3 * DB_T * NP + 4 * LN * i, g[2 * i], g[2 * i + 1]);
#pragma unroll
      for (int c = 0; c < C; c++)
#pragma unroll
        for (int i = 0; i < 2 * R4; i++) s[c][i] = x2_mul(s[c][i], g[i]);
    }
    int n = C * 2 * DB_T;
#pragma unroll
    for (int o = LN / 2; o > 0; o >>= 1) {
      n >>= 1;
#pragma unroll
      for (int i = 0; i < C * DB_T; i++)
        if (i < n) val[i] += __shfl_xor_sync(0xffffffffu, val[i + n], o);
    }
    const float e = v - val[0];
    const float e0 = __shfl_sync(0xffffffffu, e, first), e1 = __shfl_sync(0xffffffffu, e, first + 1), e2 = __shfl_sync(0xffffffffu, e, first + 2),
                e3 = __shfl_sync(0xffffffffu, e, first + 3);
    const float u0 = be.x * e0, u1 = be.y * fmaf(-a0.x, u0, e1), u2 = be.z * fmaf(-a0.z, u1, fmaf(-a0.y, u0, e2)),
                u3 = be.w * fmaf(-a1.y, u2, fmaf(-a1.x, u1, fmaf(-a0.w, u0, e3)));
    if (my_t == 0) {
      *reinterpret_cast<float4 *>(&su[warp][lane >> 2][0]) = make_float4(u0, u0, u1, u1);
      *reinterpret_cast<float4 *>(&su[warp][lane >> 2][2]) = make_float4(u2, u2, u3, u3);
    }
    __syncwarp();
    if (left > 0) *o_ptr = fmaf(b.w, u3, fmaf(b.z, u2, fmaf(b.y, u1, fmaf(b.x, u0, val[1]))));
    o_ptr += step;
    left -= DB_T;
    f32x2 u[C][DB_T];
#pragma unroll
    for (int c = 0; c < C; c++)
#pragma unroll
      for (int t = 0; t < DB_T; t += 2) {
        const ulonglong2 uu = *reinterpret_cast<const ulonglong2 *>(&su[warp][col_of(c)][t]);
        u[c][t] = uu.x; u[c][t + 1] = uu.y;
      }
#pragma unroll
    for (int t = 0; t < DB_T; t++) {
      f32x2 x[2 * R4];
#pragma unroll
      for (int i = 0; i < 2 * R4; i++)
        if constexpr (EARLY) x[i] = kx[t][i];
      if constexpr (!EARLY) {
#pragma unroll
        for (int i = 0; i < R4; i++) x2_load4(vec + (2 * DB_T + t) * NP + 4 * LN * i, x[2 * i], x[2 * i + 1]);
      }
#pragma unroll
      for (int c = 0; c < C; c++)
#pragma unroll
        for (int i = 0; i < 2 * R4; i++) s[c][i] = x2_fma(x[i], u[c][t], s[c][i]);
    }
    // (su is rewritten behind the next block's barrier)
  }
#pragma unroll
  for (int c = 0; c < C; c++)
#pragma unroll
    for (int i = 0; i < R4; i++)
      if (c0 + col_of(c) < V) x2_store4(S + (size_t)col_of(c) * NP + 4 * LN * i, s[c][2 * i], s[c][2 * i + 1]);
}

template <int NV>
dp_status launch_step(dp_ctx *ctx, const float *proj, int proj_stride, const DeltaShape &sh, const DeltaWeights &w, const SsmState &st, float *out, float *gate,
                      int rows, const int *pos) {
  const int limit = 100 * 1024;  // two CTAs per SM
  const dim3 grid(sh.heads, (sh.vdim + DL_COLS - 1) / DL_COLS, rows);
  if constexpr (NV <= 4)
    if (w.a2_stride <= 128 && w.g2_stride <= 128) {
      const DeltaStepSmem m = delta_step_smem(sh, w.a2_stride, w.g2_stride, limit, false);
      DP_LAUNCH(ctx, (delta_step_kernel<NV, true>), grid, DL_THREADS, (size_t)m.total, proj, proj_stride, sh, w, st, out, gate, pos, m);
      return DP_OK;
    }
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    DP_CUDA(ctx, cudaFuncSetAttribute((delta_step_kernel<NV, false>), cudaFuncAttributeMaxDynamicSharedMemorySize, limit));
    attr.done(ctx->device);
  }
  const DeltaStepSmem m = delta_step_smem(sh, w.a2_stride, w.g2_stride, limit, true);
  if (m.total > limit) return dp_fail(ctx, DP_ERR_UNSUPPORTED, "delta: low-rank sizes %d and %d exceed shared memory", sh.decay_rank, sh.gate_rank);
  DP_LAUNCH(ctx, (delta_step_kernel<NV, false>), grid, DL_THREADS, (size_t)m.total, proj, proj_stride, sh, w, st, out, gate, pos, m);
  return DP_OK;
}

template <int NV>
dp_status launch_scan(dp_ctx *ctx, const DeltaShape &sh, const SsmState &st, const DeltaRows &r, float *out, int rows, const RowMap &map) {
  constexpr int NP = 32 * NV, LN = NP >= 128 ? 32 : NP / 4;
  const size_t smem = (size_t)DS_STAGES * db_record(NP) * 4;
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    DP_CUDA(ctx, cudaFuncSetAttribute((delta_scan_kernel<NP, LN>), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr.done(ctx->device);
  }
  const int units = (rows + DB_T - 1) / DB_T * sh.heads;
  DP_LAUNCH(ctx, delta_block_kernel<NP>, (units + 3) / 4, 128, 0, sh, r, rows);
  DP_LAUNCH(ctx, (delta_scan_kernel<NP, LN>), dim3(sh.heads, (sh.vdim + DS_COLS - 1) / DS_COLS), DS_THREADS, smem, sh, st, r, out, rows, map.start_pos, map.seq);
  return DP_OK;
}

template <int JV>
dp_status launch_rows4(dp_ctx *ctx, const float *proj, int proj_stride, const DeltaShape &sh, const DeltaWeights &w, const SsmState &st, const DeltaRows &r, int rows,
                       const RowMap &map) {
  const int v_units = (sh.inner() + 127) / 128, units = sh.kv_heads + v_units + DR_AUX;
  const dim3 grid((units + 3) / 4, (rows + DR_ROWS - 1) / DR_ROWS);
#define DP_ROWS4(T) do { \
    if (r.a_low) DP_LAUNCH(ctx, (delta_rows4_kernel<JV, T, true>), grid, 128, 0, proj, proj_stride, sh, w, st, r, v_units, rows, map.start_pos, map.seq); \
    else DP_LAUNCH(ctx, (delta_rows4_kernel<JV, T, false>), grid, 128, 0, proj, proj_stride, sh, w, st, r, v_units, rows, map.start_pos, map.seq); \
  } while (0)
  switch (sh.taps) {
    case 1: DP_ROWS4(1); break;
    case 2: DP_ROWS4(2); break;
    case 3: DP_ROWS4(3); break;
    default: DP_ROWS4(4); break;
  }
#undef DP_ROWS4
  return DP_OK;
}

template <int NJ>
dp_status launch_rows(dp_ctx *ctx, const float *proj, int proj_stride, const DeltaShape &sh, const DeltaWeights &w, const SsmState &st, const DeltaRows &r, int rows,
                      const RowMap &map) {
  if (sh.taps <= 4 && sh.dim % 4 == 0 && sh.inner() % 4 == 0 && proj_stride % 4 == 0 && NJ <= 8)
    return launch_rows4<(NJ > 4 ? 2 : 1)>(ctx, proj, proj_stride, sh, w, st, r, rows, map);
  const int v_units = (sh.inner() + 32 * NJ - 1) / (32 * NJ), units = sh.kv_heads + v_units + DR_AUX;
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
size_t dpk_delta_record_floats(const DeltaShape &sh, int rows) { return (size_t)((rows + DB_T - 1) / DB_T) * sh.heads * db_record(sh.state_stride); }
