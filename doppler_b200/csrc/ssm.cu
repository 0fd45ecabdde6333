// Mamba-2 recurrence (state-space duality form) in f32:
//   S_t = exp(-exp(a_log) dt_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,   then y_t * silu(z_t)
// with x, B and C through a causal depthwise convolution and silu first, dt = softplus(dt + bias), B and C shared by
// the heads of a group.
//
// The same kernels run linear attention with a constant decay per head (see SsmShape): no convolution, step size 1.
//
// State layout: [head][vdim][state_stride], the state index fastest and padded with zeros to 32 * 2^k, so that eight
// lanes cover a column of the state with 16-byte pieces (lane s holds n = 4 s + 32 i + {0..3}) and reduce y over the
// state with three shuffles.  A sequence at position 0 starts from zeros whatever its slot held before.
#include "layers.h"
#include "pdl.cuh"

namespace {

constexpr int SSM_COLS = 32, SSM_LANES = 8, SSM_THREADS = SSM_COLS * SSM_LANES;

__device__ __forceinline__ float ssm_silu(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float ssm_softplus(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }

// ---- one token per row, rows are sequences: grid (heads, column tiles, rows) ----
// What earlier steps left (state, convolution histories, positions) is read before griddepcontrol.wait; after it only
// this token's projections are.
template <int NV>
__global__ void __launch_bounds__(SSM_THREADS) ssm_step_kernel(const float *__restrict__ proj, int proj_stride, const SsmShape sh, const SsmWeights w,
                                                               const SsmState st, float *__restrict__ out, const int *__restrict__ pos_arr) {
  constexpr int NP = NV * 32, CHANNELS = 2 * NP + SSM_COLS, PER = (CHANNELS + SSM_THREADS - 1) / SSM_THREADS;
  __shared__ __align__(16) float sv[CHANNELS];  // B, C, x
  const int tid = threadIdx.x, h = blockIdx.x, p0 = blockIdx.y * SSM_COLS, row = blockIdx.z;
  const int P = sh.vdim, N = sh.state, G = sh.groups, inner = sh.heads * P, CH = inner + 2 * G * N, taps = sh.taps;
  const int per = sh.heads / G, g = h / per;
  const int pos = pos_arr[row];
  const float *pr = proj + (size_t)row * proj_stride;
  const float *raw = pr + inner;
  float *hist = st.hist + (size_t)row * st.hist_seq;
  float *slot = hist + (size_t)(pos % taps) * CH;
  const int cols = min(SSM_COLS, P - p0);
  const bool keep_bc = blockIdx.y == 0 && h == g * per;  // one head of the group appends its B and C
  const int col = tid / SSM_LANES, sub = tid % SSM_LANES;
  float4 *S = reinterpret_cast<float4 *>(st.s + (size_t)row * st.s_seq + ((size_t)h * P + p0 + col) * NP) + sub;
  float4 v[NV];
#pragma unroll
  for (int i = 0; i < NV; i++) v[i] = (col < cols && pos > 0) ? S[8 * i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  // this thread's channels of the convolution: what the history and the bias contribute
  float acc[PER], last[PER];
  int chan[PER];
#pragma unroll
  for (int j = 0; j < PER; j++) {
    const int i = tid + j * SSM_THREADS;
    int ch = -1;
    if (i < 2 * NP) {
      const int n = i < NP ? i : i - NP;
      if (n < N) ch = inner + (i < NP ? g : G + g) * N + n;
    } else if (i < 2 * NP + cols) ch = h * P + p0 + i - 2 * NP;
    chan[j] = ch;
    acc[j] = last[j] = 0.0f;
    if (ch >= 0) {
      const float *cw = w.conv + (size_t)ch * taps;
      if (w.conv) acc[j] = w.conv_b[ch];
      last[j] = w.conv ? cw[taps - 1] : 1.0f;
      for (int k = taps - 1; k > 0; k--)
        if (pos - k >= 0) acc[j] = fmaf(cw[taps - 1 - k], hist[(size_t)((pos - k) % taps) * CH + ch], acc[j]);
    }
  }
  const float a = w.a[h], dt_bias = w.decay ? 0.0f : w.dt_bias[h], dh = w.d ? w.d[h] : 0.0f, fixed = w.decay ? w.decay[h] : 0.0f;
  pdl_wait();
  pdl_launch();
  const float dt_raw = w.decay ? 0.0f : pr[inner + CH + h];
  const int e = h * P + p0 + col;
  const float z = sub == 0 && col < cols && sh.gated ? pr[e] : 0.0f;
#pragma unroll
  for (int j = 0; j < PER; j++) {
    const int i = tid + j * SSM_THREADS;
    if (i < CHANNELS) {
      float val = 0.0f;
      if (chan[j] >= 0) {
        const float cur = raw[chan[j]];
        val = ssm_silu(fmaf(last[j], cur, acc[j]));
        if (taps > 1 && (i >= 2 * NP || keep_bc)) slot[chan[j]] = cur;
      }
      sv[i] = val;
    }
  }
  const float dt = w.decay ? 1.0f : ssm_softplus(dt_raw + dt_bias), decay = w.decay ? fixed : expf(a * dt);
  __syncthreads();
  const float x = sv[2 * NP + col], xdt = dt * x;
  float y = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const float4 b = *reinterpret_cast<const float4 *>(sv + sub * 4 + 32 * i), c = *reinterpret_cast<const float4 *>(sv + NP + sub * 4 + 32 * i);
    v[i].x = fmaf(decay, v[i].x, xdt * b.x); v[i].y = fmaf(decay, v[i].y, xdt * b.y);
    v[i].z = fmaf(decay, v[i].z, xdt * b.z); v[i].w = fmaf(decay, v[i].w, xdt * b.w);
    y = fmaf(v[i].x, c.x, fmaf(v[i].y, c.y, fmaf(v[i].z, c.z, fmaf(v[i].w, c.w, y))));
    if (col < cols) S[8 * i] = v[i];
  }
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (sub == 0 && col < cols) out[(size_t)row * inner + e] = sh.gated ? fmaf(dh, x, y) * ssm_silu(z) : fmaf(dh, x, y);
}

// ---- several tokens of one sequence: convolution and step sizes ----
constexpr int CONV_ROWS = 16;
__device__ __forceinline__ void conv_store(float *p, float v) { *p = v; }
__device__ __forceinline__ void conv_store(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void conv_store4(float *p, const float (&v)[4]) { *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void conv_store4(__nv_bfloat16 *p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
}

// an activation that is stored as bf16 needs no exact division
template <typename OutT> __device__ __forceinline__ float conv_silu(float v) {
  if constexpr (sizeof(OutT) == 2) return __fdividef(v, 1.0f + __expf(-v));
  else return ssm_silu(v);
}

// step size of one (row, head)
__device__ __forceinline__ void conv_dt(const float *proj, int proj_stride, const SsmShape &sh, const SsmWeights &w, int col0, int h, float *dt, int r0, int r1) {
  for (int r = r0; r < r1; r++) dt[(size_t)r * sh.heads + h] = ssm_softplus(proj[(size_t)r * proj_stride + col0 + h] + w.dt_bias[h]);
}

// up to four taps, four neighbouring channels per thread (channel counts and row strides that are multiples of four)
template <int TAPS, typename OutT>
__global__ void __launch_bounds__(128) ssm_conv4_kernel(const float *__restrict__ proj, int proj_stride, const SsmShape sh, const SsmWeights w, const SsmState st,
                                                        OutT *__restrict__ xbc, float *__restrict__ dt, int rows, int start_pos, int seq) {
  pdl_launch();
  pdl_wait();
  const int inner = sh.heads * sh.vdim, CH = inner + 2 * sh.groups * sh.state;
  const int idx = blockIdx.x * 128 + threadIdx.x, ch = idx * 4;
  const int r0 = blockIdx.y * CONV_ROWS, r1 = min(r0 + CONV_ROWS, rows);
  if (ch >= CH) {
    const int h = idx - CH / 4;
    if (h < sh.heads && w.dt_bias) conv_dt(proj, proj_stride, sh, w, inner + CH, h, dt, r0, r1);
    return;
  }
  const float *col = proj + inner + ch;
  const float *hist = st.hist + (size_t)seq * st.hist_seq;
  auto raw = [&](int r) -> float4 {
    if (r >= 0) return *reinterpret_cast<const float4 *>(col + (size_t)r * proj_stride);
    const int p = start_pos + r;
    return p >= 0 ? *reinterpret_cast<const float4 *>(hist + (size_t)(p % TAPS) * CH + ch) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  };
  float wv[4][TAPS], bias[4];  // the taps of each channel
#pragma unroll
  for (int i = 0; i < 4; i++) {
    bias[i] = w.conv ? w.conv_b[ch + i] : 0.0f;
    if constexpr (TAPS == 4) {
      const float4 v = *reinterpret_cast<const float4 *>(w.conv + (size_t)(ch + i) * 4);
      wv[i][0] = v.x; wv[i][1] = v.y; wv[i][2] = v.z; wv[i][3] = v.w;
    } else {
#pragma unroll
      for (int k = 0; k < TAPS; k++) wv[i][k] = w.conv ? w.conv[(size_t)(ch + i) * TAPS + k] : 1.0f;
    }
  }
  float4 win[TAPS];  // rows r - (TAPS - 1) .. r
#pragma unroll
  for (int k = 0; k + 1 < TAPS; k++) win[k + 1] = raw(r0 - (TAPS - 1) + k);
#pragma unroll 8
  for (int r = r0; r < r1; r++) {
#pragma unroll
    for (int k = 0; k + 1 < TAPS; k++) win[k] = win[k + 1];
    win[TAPS - 1] = *reinterpret_cast<const float4 *>(col + (size_t)r * proj_stride);
    float o[4] = {bias[0], bias[1], bias[2], bias[3]};
#pragma unroll
    for (int k = 0; k < TAPS; k++) {
      o[0] = fmaf(wv[0][k], win[k].x, o[0]); o[1] = fmaf(wv[1][k], win[k].y, o[1]);
      o[2] = fmaf(wv[2][k], win[k].z, o[2]); o[3] = fmaf(wv[3][k], win[k].w, o[3]);
    }
#pragma unroll
    for (int i = 0; i < 4; i++) o[i] = conv_silu<OutT>(o[i]);
    conv_store4(xbc + (size_t)r * CH + ch, o);
    if (TAPS > 1 && r >= rows - (TAPS - 1)) *reinterpret_cast<float4 *>(st.stage + (size_t)((start_pos + r) % TAPS) * CH + ch) = win[TAPS - 1];
  }
}

// any number of taps and channels
template <typename OutT>
__global__ void __launch_bounds__(128) ssm_conv_kernel(const float *__restrict__ proj, int proj_stride, const SsmShape sh, const SsmWeights w, const SsmState st,
                                                       OutT *__restrict__ xbc, float *__restrict__ dt, int rows, int start_pos, int seq) {
  pdl_launch();
  pdl_wait();
  const int inner = sh.heads * sh.vdim, CH = inner + 2 * sh.groups * sh.state, taps = sh.taps;
  const int ch = blockIdx.x * 128 + threadIdx.x;
  const int r0 = blockIdx.y * CONV_ROWS, r1 = min(r0 + CONV_ROWS, rows);
  if (ch >= CH) {
    if (ch < CH + sh.heads && w.dt_bias) conv_dt(proj, proj_stride, sh, w, inner + CH, ch - CH, dt, r0, r1);
    return;
  }
  const float *col = proj + inner + ch;
  const float *hist = st.hist + (size_t)seq * st.hist_seq;
  auto raw = [&](int r) -> float {
    if (r >= 0) return col[(size_t)r * proj_stride];
    const int p = start_pos + r;
    return p >= 0 ? hist[(size_t)(p % taps) * CH + ch] : 0.0f;
  };
  const float *cw = w.conv + (size_t)ch * taps;
  for (int r = r0; r < r1; r++) {
    float acc = w.conv ? w.conv_b[ch] : raw(r);
    if (w.conv)
      for (int j = 0; j < taps; j++) acc = fmaf(cw[j], raw(r - (taps - 1) + j), acc);
    conv_store(xbc + (size_t)r * CH + ch, conv_silu<OutT>(acc));
    if (r >= rows - (taps - 1)) st.stage[(size_t)((start_pos + r) % taps) * CH + ch] = raw(r);
  }
}

// ---- several tokens of one sequence, token by token: grid (heads, column tiles) ----
constexpr int SCAN_TB = 16;  // tokens staged at a time
__device__ __forceinline__ void scan_cp4(float *dst, const float *src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
template <int NV>
__global__ void __launch_bounds__(SSM_THREADS) ssm_scan_kernel(const float *__restrict__ proj, int proj_stride, const float *__restrict__ xbc,
                                                               const float *__restrict__ dt, const SsmShape sh, const SsmWeights w, const SsmState st,
                                                               float *__restrict__ out, int rows, int start_pos, int seq) {
  pdl_launch();
  pdl_wait();
  constexpr int NP = NV * 32, TOK = 2 * NP + SSM_COLS + 4;  // floats staged per token: B, C, x, dt
  extern __shared__ __align__(16) float scan_smem[];         // [2][SCAN_TB][TOK], then y [SCAN_TB][SSM_COLS]
  float *sy = scan_smem + 2 * SCAN_TB * TOK;
  const int tid = threadIdx.x, h = blockIdx.x, p0 = blockIdx.y * SSM_COLS;
  const int P = sh.vdim, N = sh.state, G = sh.groups, inner = sh.heads * P, CH = inner + 2 * G * N;
  const int g = h / (sh.heads / G), cols = min(SSM_COLS, P - p0);
  const int col = tid / SSM_LANES, sub = tid % SSM_LANES;
  for (int i = tid; i < 2 * SCAN_TB * TOK; i += SSM_THREADS) scan_smem[i] = 0.0f;  // padded state columns stay zero
  __syncthreads();
  auto stage = [&](int blk) {
    float *dst = scan_smem + (blk & 1) * SCAN_TB * TOK;
    const int r0 = blk * SCAN_TB, n = min(SCAN_TB, rows - r0);
    const int per = 2 * N + cols + (w.decay ? 0 : 1);
    for (int i = tid; i < n * per; i += SSM_THREADS) {
      const int t = i / per, e = i - t * per;
      const float *src = xbc + (size_t)(r0 + t) * CH;
      float *d = dst + t * TOK;
      if (e < N) scan_cp4(d + e, src + inner + g * N + e);
      else if (e < 2 * N) scan_cp4(d + NP + e - N, src + inner + (G + g) * N + e - N);
      else if (e < 2 * N + cols) scan_cp4(d + 2 * NP + e - 2 * N, src + h * P + p0 + e - 2 * N);
      else scan_cp4(d + 2 * NP + SSM_COLS, dt + (size_t)(r0 + t) * sh.heads + h);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float4 v[NV];
  float4 *S = reinterpret_cast<float4 *>(st.s + (size_t)seq * st.s_seq + ((size_t)h * P + p0 + col) * NP) + sub;
#pragma unroll
  for (int i = 0; i < NV; i++) v[i] = (col < cols && start_pos > 0) ? S[8 * i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  const float a = w.a[h], dh = w.d ? w.d[h] : 0.0f, fixed = w.decay ? w.decay[h] : 0.0f;
  const int blocks = (rows + SCAN_TB - 1) / SCAN_TB;
  stage(0);
  for (int blk = 0; blk < blocks; blk++) {
    if (blk + 1 < blocks) {
      stage(blk + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float *src = scan_smem + (blk & 1) * SCAN_TB * TOK;
    const int r0 = blk * SCAN_TB, n = min(SCAN_TB, rows - r0);
#pragma unroll 2
    for (int t = 0; t < n; t++) {
      const float *d = src + t * TOK;
      const float step = w.decay ? 1.0f : d[2 * NP + SSM_COLS], decay = w.decay ? fixed : expf(a * step), x = d[2 * NP + col], xdt = step * x;
      float y = 0.0f;
#pragma unroll
      for (int i = 0; i < NV; i++) {
        const float4 b = *reinterpret_cast<const float4 *>(d + sub * 4 + 32 * i), c = *reinterpret_cast<const float4 *>(d + NP + sub * 4 + 32 * i);
        v[i].x = fmaf(decay, v[i].x, xdt * b.x); v[i].y = fmaf(decay, v[i].y, xdt * b.y);
        v[i].z = fmaf(decay, v[i].z, xdt * b.z); v[i].w = fmaf(decay, v[i].w, xdt * b.w);
        y = fmaf(v[i].x, c.x, fmaf(v[i].y, c.y, fmaf(v[i].z, c.z, fmaf(v[i].w, c.w, y))));
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (sub == 0) sy[t * SSM_COLS + col] = fmaf(dh, x, y);
    }
    __syncthreads();
    for (int i = tid; i < n * SSM_COLS; i += SSM_THREADS) {
      const int t = i / SSM_COLS, c = i - t * SSM_COLS;
      if (c < cols) {
        const int e = h * P + p0 + c;
        out[(size_t)(r0 + t) * inner + e] = sh.gated ? sy[i] * ssm_silu(proj[(size_t)(r0 + t) * proj_stride + e]) : sy[i];
      }
    }
  }
  if (col < cols)
#pragma unroll
    for (int i = 0; i < NV; i++) S[8 * i] = v[i];
}

template <typename KB, typename KF>
dp_status launch_conv(dp_ctx *ctx, bool bf16, KB kb, KF kf, dim3 grid, const float *proj, int proj_stride, const SsmShape &sh, const SsmWeights &w,
                      const SsmState &st, void *xbc, float *dt, int rows, const RowMap &map) {
  if (bf16) DP_LAUNCH(ctx, kb, grid, 128, 0, proj, proj_stride, sh, w, st, (__nv_bfloat16 *)xbc, dt, rows, map.start_pos, map.seq);
  else DP_LAUNCH(ctx, kf, grid, 128, 0, proj, proj_stride, sh, w, st, (float *)xbc, dt, rows, map.start_pos, map.seq);
  return DP_OK;
}

template <int NV>
dp_status launch_scan(dp_ctx *ctx, const float *proj, int proj_stride, const float *xbc, const float *dt, const SsmShape &sh, const SsmWeights &w,
                      const SsmState &st, float *out, int rows, const RowMap &map) {
  const size_t smem = (size_t)(2 * SCAN_TB * (2 * NV * 32 + SSM_COLS + 4) + SCAN_TB * SSM_COLS) * 4;
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    DP_CUDA(ctx, cudaFuncSetAttribute(ssm_scan_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr.done(ctx->device);
  }
  DP_LAUNCH(ctx, ssm_scan_kernel<NV>, dim3(sh.heads, (sh.vdim + SSM_COLS - 1) / SSM_COLS), SSM_THREADS, smem, proj, proj_stride, xbc, dt, sh, w, st, out, rows,
            map.start_pos, map.seq);
  return DP_OK;
}

}  // namespace

int dpk_ssm_state_stride(int state) {
  for (int nv = 1; nv <= 16; nv *= 2)
    if (state <= 32 * nv) return 32 * nv;
  return 0;
}

dp_status dpk_ssm_step(dp_ctx *ctx, const float *proj, int proj_stride, const SsmShape &sh, const SsmWeights &w, const SsmState &st, float *out, int rows,
                       const int *pos) {
  const dim3 grid(sh.heads, (sh.vdim + SSM_COLS - 1) / SSM_COLS, rows);
  switch (sh.state_stride / 32) {
    case 1: DP_LAUNCH(ctx, ssm_step_kernel<1>, grid, SSM_THREADS, 0, proj, proj_stride, sh, w, st, out, pos); break;
    case 2: DP_LAUNCH(ctx, ssm_step_kernel<2>, grid, SSM_THREADS, 0, proj, proj_stride, sh, w, st, out, pos); break;
    case 4: DP_LAUNCH(ctx, ssm_step_kernel<4>, grid, SSM_THREADS, 0, proj, proj_stride, sh, w, st, out, pos); break;
    case 8: DP_LAUNCH(ctx, ssm_step_kernel<8>, grid, SSM_THREADS, 0, proj, proj_stride, sh, w, st, out, pos); break;
    case 16: DP_LAUNCH(ctx, ssm_step_kernel<16>, grid, SSM_THREADS, 0, proj, proj_stride, sh, w, st, out, pos); break;
    default: return dp_fail(ctx, DP_ERR_UNSUPPORTED, "ssm: state size %d", sh.state);
  }
  return DP_OK;
}

dp_status dpk_ssm_conv(dp_ctx *ctx, const float *proj, int proj_stride, const SsmShape &sh, const SsmWeights &w, const SsmState &st, void *xbc, bool bf16,
                       float *dt, int rows, const RowMap &map) {
  const int inner = sh.heads * sh.vdim, CH = inner + 2 * sh.groups * sh.state;
  const bool four = sh.taps <= 4 && CH % 4 == 0 && inner % 4 == 0 && proj_stride % 4 == 0;
  const int threads = (four ? CH / 4 : CH) + sh.heads;
  const dim3 grid((threads + 127) / 128, (rows + CONV_ROWS - 1) / CONV_ROWS);
  if (!four) return launch_conv(ctx, bf16, ssm_conv_kernel<__nv_bfloat16>, ssm_conv_kernel<float>, grid, proj, proj_stride, sh, w, st, xbc, dt, rows, map);
#define DP_CONV(T) launch_conv(ctx, bf16, ssm_conv4_kernel<T, __nv_bfloat16>, ssm_conv4_kernel<T, float>, grid, proj, proj_stride, sh, w, st, xbc, dt, rows, map)
  switch (sh.taps) {
    case 1: return DP_CONV(1);
    case 2: return DP_CONV(2);
    case 3: return DP_CONV(3);
  }
  return DP_CONV(4);
#undef DP_CONV
}

dp_status dpk_ssm_scan(dp_ctx *ctx, const float *proj, int proj_stride, const float *xbc, const float *dt, const SsmShape &sh, const SsmWeights &w,
                       const SsmState &st, float *out, int rows, const RowMap &map) {
  switch (sh.state_stride / 32) {
    case 1: return launch_scan<1>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
    case 2: return launch_scan<2>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
    case 4: return launch_scan<4>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
    case 8: return launch_scan<8>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
    case 16: return launch_scan<16>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
  }
  return dp_fail(ctx, DP_ERR_UNSUPPORTED, "ssm: state size %d", sh.state);
}
