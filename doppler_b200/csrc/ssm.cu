// Mamba-2 recurrence (state-space duality form) in f32:
//   S_t = exp(-exp(a_log) dt_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,   then y_t * silu(z_t)
// with x, B and C through a causal depthwise convolution and silu first, dt = softplus(dt + bias), B and C shared by
// the heads of a group.
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

// convolution of channel ch of the token at `pos`, whose raw value is `cur`, over a sequence's history
__device__ __forceinline__ float ssm_conv1(const SsmWeights &w, const float *hist, int taps, int CH, int ch, int pos, float cur) {
  const float *cw = w.conv + (size_t)ch * taps;
  float acc = w.conv_b[ch];
  for (int k = taps - 1; k > 0; k--)
    if (pos - k >= 0) acc = fmaf(cw[taps - 1 - k], hist[(size_t)((pos - k) % taps) * CH + ch], acc);
  return ssm_silu(fmaf(cw[taps - 1], cur, acc));
}

// ---- one token per row, rows are sequences: grid (heads, column tiles, rows) ----
template <int NV>
__global__ void __launch_bounds__(SSM_THREADS) ssm_step_kernel(const float *__restrict__ proj, int proj_stride, const SsmShape sh, const SsmWeights w,
                                                               const SsmState st, float *__restrict__ out, const int *__restrict__ pos_arr) {
  pdl_launch();
  pdl_wait();
  constexpr int NP = NV * 32;
  __shared__ __align__(16) float sB[NP], sC[NP], sx[SSM_COLS];
  __shared__ float s_dt;
  const int tid = threadIdx.x, h = blockIdx.x, p0 = blockIdx.y * SSM_COLS, row = blockIdx.z;
  const int P = sh.vdim, N = sh.state, G = sh.groups, inner = sh.heads * P, CH = inner + 2 * G * N, taps = sh.taps;
  const int per = sh.heads / G, g = h / per;
  const int pos = pos_arr[row];
  const float *pr = proj + (size_t)row * proj_stride;
  const float *raw = pr + inner;
  float *hist = st.hist + (size_t)row * st.hist_seq;
  float *slot = hist + (size_t)(pos % taps) * CH;
  const int cols = min(SSM_COLS, P - p0);
  const bool keep_bc = taps > 1 && blockIdx.y == 0 && h == g * per;  // one head of the group appends its B and C
  // the state's first pieces are asked for while the convolution works
  const int col = tid / SSM_LANES, sub = tid % SSM_LANES;
  float4 *S = reinterpret_cast<float4 *>(st.s + (size_t)row * st.s_seq + ((size_t)h * P + p0 + col) * NP) + sub;
  float4 v[NV];
#pragma unroll
  for (int i = 0; i < NV; i++) v[i] = (col < cols && pos > 0) ? S[8 * i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  for (int i = tid; i < 2 * NP + cols; i += SSM_THREADS) {
    if (i < 2 * NP) {
      const bool is_c = i >= NP;
      const int n = is_c ? i - NP : i;
      float val = 0.0f;
      if (n < N) {
        const int ch = inner + (is_c ? G * N : 0) + g * N + n;
        const float cur = raw[ch];
        val = ssm_conv1(w, hist, taps, CH, ch, pos, cur);
        if (keep_bc) slot[ch] = cur;
      }
      (is_c ? sC : sB)[n] = val;
    } else {
      const int c = i - 2 * NP, ch = h * P + p0 + c;
      const float cur = raw[ch];
      sx[c] = ssm_conv1(w, hist, taps, CH, ch, pos, cur);
      if (taps > 1) slot[ch] = cur;
    }
  }
  if (tid == 0) s_dt = ssm_softplus(pr[inner + CH + h] + w.dt_bias[h]);
  __syncthreads();
  const float dt = s_dt, decay = expf(-expf(w.a_log[h]) * dt);
  const float x = col < cols ? sx[col] : 0.0f, xdt = dt * x;
  float y = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const float4 b = *reinterpret_cast<const float4 *>(sB + sub * 4 + 32 * i), c = *reinterpret_cast<const float4 *>(sC + sub * 4 + 32 * i);
    v[i].x = fmaf(decay, v[i].x, xdt * b.x); v[i].y = fmaf(decay, v[i].y, xdt * b.y);
    v[i].z = fmaf(decay, v[i].z, xdt * b.z); v[i].w = fmaf(decay, v[i].w, xdt * b.w);
    y = fmaf(v[i].x, c.x, fmaf(v[i].y, c.y, fmaf(v[i].z, c.z, fmaf(v[i].w, c.w, y))));
    if (col < cols) S[8 * i] = v[i];
  }
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (sub == 0 && col < cols) {
    const int e = h * P + p0 + col;
    out[(size_t)row * inner + e] = fmaf(w.d[h], x, y) * ssm_silu(pr[e]);
  }
}

// ---- several tokens of one sequence: convolution and step sizes ----
constexpr int CONV_ROWS = 16;
template <int TAPS>  // 0: any
__global__ void __launch_bounds__(128) ssm_conv_kernel(const float *__restrict__ proj, int proj_stride, const SsmShape sh, const SsmWeights w, const SsmState st,
                                                       float *__restrict__ xbc, float *__restrict__ dt, int rows, int start_pos, int seq) {
  pdl_launch();
  pdl_wait();
  const int inner = sh.heads * sh.vdim, CH = inner + 2 * sh.groups * sh.state, taps = TAPS ? TAPS : sh.taps;
  const int ch = blockIdx.x * 128 + threadIdx.x;
  const int r0 = blockIdx.y * CONV_ROWS, r1 = min(r0 + CONV_ROWS, rows);
  if (ch >= CH + sh.heads) return;
  if (ch >= CH) {
    const int h = ch - CH;
    for (int r = r0; r < r1; r++) dt[(size_t)r * sh.heads + h] = ssm_softplus(proj[(size_t)r * proj_stride + inner + ch] + w.dt_bias[h]);
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
  const float bias = w.conv_b[ch];
  if constexpr (TAPS > 0) {
    float win[TAPS], wv[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; j++) wv[j] = cw[j];
#pragma unroll
    for (int j = 0; j < TAPS - 1; j++) win[j + 1] = raw(r0 - (TAPS - 1) + j);
#pragma unroll 4
    for (int r = r0; r < r1; r++) {
#pragma unroll
      for (int j = 0; j < TAPS - 1; j++) win[j] = win[j + 1];
      win[TAPS - 1] = col[(size_t)r * proj_stride];
      float acc = bias;
#pragma unroll
      for (int j = 0; j < TAPS; j++) acc = fmaf(wv[j], win[j], acc);
      xbc[(size_t)r * CH + ch] = ssm_silu(acc);
    }
  } else {
    for (int r = r0; r < r1; r++) {
      float acc = bias;
      for (int j = 0; j < taps; j++) acc = fmaf(cw[j], raw(r - (taps - 1) + j), acc);
      xbc[(size_t)r * CH + ch] = ssm_silu(acc);
    }
  }
  if (taps > 1)
    for (int r = max(r0, rows - (taps - 1)); r < r1; r++) st.stage[(size_t)((start_pos + r) % taps) * CH + ch] = col[(size_t)r * proj_stride];
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
    const int per = 2 * N + cols + 1;
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
  const float a = -expf(w.a_log[h]), dh = w.d[h];
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
      const float step = d[2 * NP + SSM_COLS], decay = expf(a * step), x = d[2 * NP + col], xdt = step * x;
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
        out[(size_t)(r0 + t) * inner + e] = sy[i] * ssm_silu(proj[(size_t)(r0 + t) * proj_stride + e]);
      }
    }
  }
  if (col < cols)
#pragma unroll
    for (int i = 0; i < NV; i++) S[8 * i] = v[i];
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

dp_status dpk_ssm_conv(dp_ctx *ctx, const float *proj, int proj_stride, const SsmShape &sh, const SsmWeights &w, const SsmState &st, float *xbc, float *dt,
                       int rows, const RowMap &map) {
  const int cols = sh.heads * sh.vdim + 2 * sh.groups * sh.state + sh.heads;
  const dim3 grid((cols + 127) / 128, (rows + CONV_ROWS - 1) / CONV_ROWS);
  if (sh.taps == 4) DP_LAUNCH(ctx, ssm_conv_kernel<4>, grid, 128, 0, proj, proj_stride, sh, w, st, xbc, dt, rows, map.start_pos, map.seq);
  else DP_LAUNCH(ctx, ssm_conv_kernel<0>, grid, 128, 0, proj, proj_stride, sh, w, st, xbc, dt, rows, map.start_pos, map.seq);
  return DP_OK;
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
