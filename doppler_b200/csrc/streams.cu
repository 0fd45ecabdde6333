// Residual streams (hyper-connections), grouped RMSNorm and the causal input convolution of a sublayer, for several
// rows at once.  (A single decode row does all of this inside the GEMV kernels, gemv_bf16.cu.)
//
// The boundary kernel joins everything between two sublayers: x_t <- sum_s mix[s][t] x_s + out[t] y of the one that
// ended, u = sum_t in[t] x_t, RMSNorm of u per group of channels, and h + conv(h) of the next one.  A group's norm
// needs the channels of that group only, so a CTA owns (a block of rows, one group): one warp per row computes h
// into shared memory, rows before the block (the convolution's reach) are recomputed or come from the sequence's
// history, then all threads convolve.  x is read and written once per sublayer; h never goes to memory except for
// the last taps - 1 rows of a portion.
#include "layers.h"
#include "pdl.cuh"

namespace {

constexpr int SB_THREADS = 288, SB_WARPS = SB_THREADS / 32;

template <int V> struct FV { float v[V]; };
template <int V> __device__ __forceinline__ FV<V> ldv(const float *p) {
  FV<V> r;
  if constexpr (V == 4) { const float4 a = *reinterpret_cast<const float4 *>(p); r.v[0] = a.x; r.v[1] = a.y; r.v[2] = a.z; r.v[3] = a.w; }
  else r.v[0] = *p;
  return r;
}
template <int V> __device__ __forceinline__ void stv(float *p, const FV<V> &r) {
  if constexpr (V == 4) *reinterpret_cast<float4 *>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int V> __device__ __forceinline__ void stv(__nv_bfloat16 *p, const FV<V> &r) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
  } else *p = __float2bfloat16_rn(r.v[0]);
}
template <int V> __device__ __forceinline__ FV<V> ldw(const __nv_bfloat16 *p) {
  FV<V> r;
  if constexpr (V == 4) {
    const uint2 q = *reinterpret_cast<const uint2 *>(p);
    r.v[0] = __uint_as_float(q.x << 16); r.v[1] = __uint_as_float(q.x & 0xffff0000u);
    r.v[2] = __uint_as_float(q.y << 16); r.v[3] = __uint_as_float(q.y & 0xffff0000u);
    return r;
  }
#pragma unroll
  for (int i = 0; i < V; i++) r.v[i] = __bfloat162float(p[i]);
  return r;
}

struct BoundaryArgs {
  const float *x, *y;
  float *x_out;
  SublayerOut end;
  SublayerIn next;
  int streams, width, rows, dst_stride, block_rows;
  RowMap map;
};

template <int SM, int V, typename OutT>
__global__ void __launch_bounds__(SB_THREADS, 2) stream_boundary_kernel(const BoundaryArgs a, OutT *__restrict__ dst) {
  pdl_launch();
  pdl_wait();
  extern __shared__ float sb_h[];  // [halo + block_rows][gs]
  __shared__ float s_mix[SM * SM], s_out[SM], s_in[SM];
  const int S = a.streams, H = a.width, gs = H / a.next.groups, taps = a.next.taps;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const bool per_seq = a.map.pos != nullptr;
  const int halo = (per_seq || taps < 2) ? 0 : taps - 1;
  const int row0 = blockIdx.x * a.block_rows, c0 = blockIdx.y * gs;
  const int nrows = min(a.block_rows, a.rows - row0);
  for (int i = tid; i < SM; i += SB_THREADS) {
    s_in[i] = i < S ? a.next.in[i] : 0.0f;
    s_out[i] = (i < S && a.y) ? a.end.out[i] : 0.0f;
  }
  for (int i = tid; i < SM * SM; i += SB_THREADS) {
    const int s = i / SM, t = i % SM;
    s_mix[i] = (s < S && t < S && a.y) ? a.end.mix[s * S + t] : 0.0f;
  }
  __syncthreads();

  // few streams: the mixing weights in registers
  constexpr bool REG = SM <= 4;
  float r_mix[REG ? SM * SM : 1], r_out[REG ? SM : 1], r_in[REG ? SM : 1];
  if constexpr (REG) {
#pragma unroll
    for (int i = 0; i < SM * SM; i++) r_mix[i] = s_mix[i];
#pragma unroll
    for (int i = 0; i < SM; i++) { r_out[i] = s_out[i]; r_in[i] = s_in[i]; }
  }
  auto mix = [&](int s, int t) { if constexpr (REG) return r_mix[s * SM + t]; else return s_mix[s * SM + t]; };
  auto wout = [&](int t) { if constexpr (REG) return r_out[t]; else return s_out[t]; };
  auto win = [&](int t) { if constexpr (REG) return r_in[t]; else return s_in[t]; };

  // ---- h of the block's rows and of the rows the convolution reaches back to: one warp per row ----
  for (int j = warp; j < halo + nrows; j += SB_WARPS) {
    const int row = row0 + j - halo;
    float *h = sb_h + (size_t)j * gs;
    if (row < 0) {  // before this portion: the sequence's history, zeros before its start
      const int p = a.map.start_pos + row;
      const float *src = a.next.hist + (size_t)a.map.seq * a.next.hist_seq + (size_t)(p >= 0 ? p % taps : 0) * H + c0;
      for (int c = lane; c < gs; c += 32) h[c] = p >= 0 ? src[c] : 0.0f;
      continue;
    }
    const float *xr = a.x + (size_t)row * S * H + c0;
    float *xo = a.x_out + (size_t)row * S * H + c0;
    const bool store = a.y && j >= halo;
    float ss = 0.0f, y_inv = 1.0f;
    if (a.end.norm_w) {  // what the sublayer hands over passes a norm of its own
      float sy = 0.0f;
      for (int c = lane * V; c < gs; c += 32 * V) {
        const FV<V> yv = ldv<V>(a.y + (size_t)row * H + c0 + c);
#pragma unroll
        for (int i = 0; i < V; i++) sy = fmaf(yv.v[i], yv.v[i], sy);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) sy += __shfl_xor_sync(0xffffffffu, sy, o);
      y_inv = 1.0f / sqrtf(sy / (float)gs + a.end.eps);
    }
#pragma unroll(SM <= 4 ? 2 : 1)
    for (int c = lane * V; c < gs; c += 32 * V) {
      FV<V> xs[SM], u;
#pragma unroll
      for (int i = 0; i < V; i++) u.v[i] = 0.0f;
#pragma unroll
      for (int s = 0; s < SM; s++)
        if (s < S) xs[s] = ldv<V>(xr + (size_t)s * H + c);
      if (a.y) {
        FV<V> yv = ldv<V>(a.y + (size_t)row * H + c0 + c);
        if (a.end.norm_w) {
          const FV<V> w = ldw<V>(a.end.norm_w + c0 + c);
#pragma unroll
          for (int i = 0; i < V; i++) yv.v[i] = yv.v[i] * y_inv * w.v[i];
        }
#pragma unroll
        for (int t = 0; t < SM; t++) {
          if (t < S) {
            FV<V> n;
#pragma unroll
            for (int i = 0; i < V; i++) n.v[i] = wout(t) * yv.v[i];
#pragma unroll
            for (int s = 0; s < SM; s++)
              if (s < S)
#pragma unroll
                for (int i = 0; i < V; i++) n.v[i] = fmaf(mix(s, t), xs[s].v[i], n.v[i]);
            if (store) stv<V>(xo + (size_t)t * H + c, n);
#pragma unroll
            for (int i = 0; i < V; i++) u.v[i] = fmaf(win(t), n.v[i], u.v[i]);
          }
        }
      } else {
#pragma unroll
        for (int s = 0; s < SM; s++)
          if (s < S)
#pragma unroll
            for (int i = 0; i < V; i++) u.v[i] = fmaf(win(s), xs[s].v[i], u.v[i]);
      }
#pragma unroll
      for (int i = 0; i < V; i++) ss = fmaf(u.v[i], u.v[i], ss);
      stv<V>(h + c, u);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = 1.0f / sqrtf(ss / (float)gs + a.next.eps);
    for (int c = lane * V; c < gs; c += 32 * V) {
      FV<V> v = ldv<V>(h + c);
      const FV<V> w = ldw<V>(a.next.norm_w + c0 + c);
#pragma unroll
      for (int i = 0; i < V; i++) v.v[i] = v.v[i] * inv * w.v[i];
      stv<V>(h + c, v);
    }
  }
  __syncthreads();

  // ---- h + conv(h), the sublayer's input; the rows later tokens reach back to ----
  const int cv = gs / V;
  for (int idx = tid; idx < nrows * cv; idx += SB_THREADS) {
    const int r = idx / cv, c = (idx - r * cv) * V, row = row0 + r;
    const FV<V> h = ldv<V>(sb_h + (size_t)(halo + r) * gs + c);
    FV<V> o = h;
    if (taps > 0) {
      const __nv_bfloat16 *w = a.next.conv_w + (size_t)(c0 + c) * taps;
      const int pos = per_seq ? a.map.pos[row] : a.map.start_pos + row;
      FV<V> acc;
#pragma unroll
      for (int i = 0; i < V; i++) acc.v[i] = 0.0f;
      for (int k = taps - 1; k > 0; k--) {  // k positions back
        FV<V> past;
        if (per_seq) {
#pragma unroll
          for (int i = 0; i < V; i++) past.v[i] = 0.0f;
          if (pos - k >= 0) past = ldv<V>(a.next.hist + (size_t)row * a.next.hist_seq + (size_t)((pos - k) % taps) * H + c0 + c);
        } else {
          past = ldv<V>(sb_h + (size_t)(halo + r - k) * gs + c);
        }
#pragma unroll
        for (int i = 0; i < V; i++) acc.v[i] = fmaf(__bfloat162float(w[i * taps + taps - 1 - k]), past.v[i], acc.v[i]);
      }
#pragma unroll
      for (int i = 0; i < V; i++) o.v[i] = h.v[i] + fmaf(__bfloat162float(w[i * taps + taps - 1]), h.v[i], acc.v[i]);
      if (taps > 1) {
        if (per_seq) stv<V>(a.next.hist + (size_t)row * a.next.hist_seq + (size_t)(pos % taps) * H + c0 + c, h);
        else if (row >= a.rows - (taps - 1)) stv<V>(a.next.stage + (size_t)(pos % taps) * H + c0 + c, h);
      }
    }
    stv<V>(dst + (size_t)row * a.dst_stride + c0 + c, o);
  }
}

template <int SM, int V>
dp_status launch_boundary(dp_ctx *ctx, const BoundaryArgs &a, void *dst, bool bf16, dim3 grid, size_t smem) {
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    const int cap = (int)ctx->smem_optin - 4096;  // beside the kernel's static shared memory
    DP_CUDA(ctx, cudaFuncSetAttribute((stream_boundary_kernel<SM, V, float>), cudaFuncAttributeMaxDynamicSharedMemorySize, cap));
    DP_CUDA(ctx, cudaFuncSetAttribute((stream_boundary_kernel<SM, V, __nv_bfloat16>), cudaFuncAttributeMaxDynamicSharedMemorySize, cap));
    attr.done(ctx->device);
  }
  if (bf16) DP_LAUNCH(ctx, (stream_boundary_kernel<SM, V, __nv_bfloat16>), grid, SB_THREADS, smem, a, (__nv_bfloat16 *)dst);
  else DP_LAUNCH(ctx, (stream_boundary_kernel<SM, V, float>), grid, SB_THREADS, smem, a, (float *)dst);
  return DP_OK;
}

// One stream, one norm group, no input convolution: a CTA per row, the row in registers (at most 4 * 256 * MAXV values).
// x_out (optional) <- mix x + out norm(y); dst (optional) <- RMSNorm of that.
template <int MAXV, typename OutT>
__global__ void __launch_bounds__(256) stream_row_kernel(const float *__restrict__ x, float *__restrict__ x_out, const float *__restrict__ y, const SublayerOut end,
                                                         const SublayerIn next, int H, OutT *__restrict__ dst, int dst_stride) {
  pdl_launch();
  pdl_wait();
  __shared__ float sh[16];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const size_t base = (size_t)blockIdx.x * H;
  auto block_sum = [&](float v, float *red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; i++) t += red[i];
    return t;
  };
  FV<4> v[MAXV], yv[MAXV];
#pragma unroll
  for (int j = 0; j < MAXV; j++) {
    const int c = (tid + 256 * j) * 4;
    v[j] = c < H ? ldv<4>(x + base + c) : FV<4>{};
    yv[j] = y && c < H ? ldv<4>(y + base + c) : FV<4>{};
  }
  if (y) {
    float y_inv = 1.0f;
    if (end.norm_w) {
      float sy = 0.0f;
#pragma unroll
      for (int j = 0; j < MAXV; j++)
#pragma unroll
        for (int i = 0; i < 4; i++) sy = fmaf(yv[j].v[i], yv[j].v[i], sy);
      y_inv = 1.0f / sqrtf(block_sum(sy, sh) / (float)H + end.eps);
    }
    const float mix = end.mix[0], out = end.out[0];
#pragma unroll
    for (int j = 0; j < MAXV; j++) {
      const int c = (tid + 256 * j) * 4;
      if (c < H) {
        FV<4> w = {{1.0f, 1.0f, 1.0f, 1.0f}};
        if (end.norm_w) w = ldw<4>(end.norm_w + c);
#pragma unroll
        for (int i = 0; i < 4; i++) v[j].v[i] = fmaf(mix, v[j].v[i], out * (yv[j].v[i] * y_inv * w.v[i]));
        if (x_out) stv<4>(x_out + base + c, v[j]);
      }
    }
  }
  if (!dst) return;
  float ss = 0.0f;
  const float in = next.in[0];
#pragma unroll
  for (int j = 0; j < MAXV; j++)
#pragma unroll
    for (int i = 0; i < 4; i++) {
      v[j].v[i] *= in;
      ss = fmaf(v[j].v[i], v[j].v[i], ss);
    }
  const float inv = 1.0f / sqrtf(block_sum(ss, sh + 8) / (float)H + next.eps);
#pragma unroll
  for (int j = 0; j < MAXV; j++) {
    const int c = (tid + 256 * j) * 4;
    if (c < H) {
      const FV<4> w = ldw<4>(next.norm_w + c);
#pragma unroll
      for (int i = 0; i < 4; i++) v[j].v[i] = v[j].v[i] * inv * w.v[i];
      stv<4>(dst + (size_t)blockIdx.x * dst_stride + c, v[j]);
    }
  }
}

template <typename OutT>
dp_status launch_row(dp_ctx *ctx, const float *x, float *x_out, const float *y, const SublayerOut &end, const SublayerIn &next, int H, OutT *dst, int dst_stride,
                     int rows) {
  if (H <= 1024) DP_LAUNCH(ctx, (stream_row_kernel<1, OutT>), rows, 256, 0, x, x_out, y, end, next, H, dst, dst_stride);
  else if (H <= 2048) DP_LAUNCH(ctx, (stream_row_kernel<2, OutT>), rows, 256, 0, x, x_out, y, end, next, H, dst, dst_stride);
  else if (H <= 4096) DP_LAUNCH(ctx, (stream_row_kernel<4, OutT>), rows, 256, 0, x, x_out, y, end, next, H, dst, dst_stride);
  else DP_LAUNCH(ctx, (stream_row_kernel<8, OutT>), rows, 256, 0, x, x_out, y, end, next, H, dst, dst_stride);
  return DP_OK;
}

// the streams' sum of a row after y has been written into them, y through its grouped norm: one CTA per row
__global__ void __launch_bounds__(256) stream_sum_norm_kernel(const float *__restrict__ x, const float *__restrict__ y, const SublayerOut end, int S, int H,
                                                              float *__restrict__ h) {
  pdl_launch();
  pdl_wait();
  __shared__ float red[8], s_inv;
  const int tid = threadIdx.x, gs = H / end.groups;
  const float *yr = y + (size_t)blockIdx.x * H;
  float w_out = 0.0f;
  for (int t = 0; t < S; t++) w_out += end.out[t];
  for (int g = 0; g < end.groups; g++) {
    float sy = 0.0f;
    for (int c = tid; c < gs; c += 256) sy = fmaf(yr[g * gs + c], yr[g * gs + c], sy);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sy += __shfl_xor_sync(0xffffffffu, sy, o);
    if ((tid & 31) == 0) red[tid >> 5] = sy;
    __syncthreads();
    if (tid == 0) {
      float t = 0.0f;
      for (int i = 0; i < 8; i++) t += red[i];
      s_inv = 1.0f / sqrtf(t / (float)gs + end.eps);
    }
    __syncthreads();
    for (int c = g * gs + tid; c < (g + 1) * gs; c += 256) {
      float v = w_out * (yr[c] * s_inv * __bfloat162float(end.norm_w[c]));
      for (int s = 0; s < S; s++) {
        float m = 0.0f;
        for (int t = 0; t < S; t++) m += end.mix[s * S + t];
        v = fmaf(m, x[((size_t)blockIdx.x * S + s) * H + c], v);
      }
      h[(size_t)blockIdx.x * H + c] = v;
    }
    __syncthreads();
  }
}

__global__ void __launch_bounds__(256) stream_sum_kernel(const float *__restrict__ x, const float *__restrict__ y, const SublayerOut end, int S, int H,
                                                         float *__restrict__ h, int rows) {
  pdl_launch();
  pdl_wait();
  __shared__ float s_w[DP_MAX_STREAMS], s_o;
  // sum_t (sum_s mix[s][t] x_s + out[t] y) = sum_s (sum_t mix[s][t]) x_s + (sum_t out[t]) y
  if (threadIdx.x < (unsigned)S) {
    float w = 0.0f;
    for (int t = 0; t < S; t++) w += end.mix[threadIdx.x * S + t];
    s_w[threadIdx.x] = w;
  }
  if (threadIdx.x == 32) {
    float o = 0.0f;
    for (int t = 0; t < S; t++) o += end.out[t];
    s_o = o;
  }
  __syncthreads();
  const size_t total = (size_t)rows * H;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t r = i / H, c = i - r * H;
    float v = s_o * y[i];
    for (int s = 0; s < S; s++) v = fmaf(s_w[s], x[(r * S + s) * H + c], v);
    h[i] = v;
  }
}

__global__ void __launch_bounds__(256) stream_embed_kernel(const int *__restrict__ ids, const __nv_bfloat16 *__restrict__ table, int table_stride, float scale,
                                                           int S, int H, float *__restrict__ x, const float *__restrict__ in, float *__restrict__ u, int rows) {
  pdl_wait();
  pdl_launch();
  float w = 0.0f;
  if (u) for (int s = 0; s < S; s++) w += in[s];
  const size_t total = (size_t)rows * H;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t r = i / H, c = i - r * H;
    const float v = __bfloat162float(table[(size_t)ids[r] * table_stride + c]) * scale;
    for (int s = 0; s < S; s++) x[(r * S + s) * H + c] = v;
    if (u) u[i] = w * v;
  }
}

template <int V> __device__ __forceinline__ void gate_by(FV<V> &v, const float *gate) {
  const FV<V> g = ldv<V>(gate);
#pragma unroll
  for (int i = 0; i < V; i++) v.v[i] *= 1.0f / (1.0f + expf(-g.v[i]));
}

// one warp per (row, part), the part in registers (parts of at most 128 * MAXV values, all sizes multiples of four)
template <int MAXV, typename OutT>
__global__ void __launch_bounds__(256) group_norm_warp_kernel(const float *__restrict__ x, int x_stride, const GroupNorm n, int gs, OutT *__restrict__ dst,
                                                              int dst_stride, int rows) {
  pdl_launch();
  pdl_wait();
  const int groups = n.groups;
  const int lane = threadIdx.x & 31, part = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (part >= rows * groups) return;
  const int row = part / groups, c0 = (part - row * groups) * gs;
  const float *xr = x + (size_t)row * x_stride + c0;
  FV<4> v[MAXV];
  float ss = 0.0f;
#pragma unroll
  for (int j = 0; j < MAXV; j++) {
    const int c = (lane + 32 * j) * 4;
    if (c < gs) v[j] = ldv<4>(xr + c);
    else v[j] = FV<4>{};
  }
#pragma unroll
  for (int j = 0; j < MAXV; j++)
#pragma unroll
    for (int i = 0; i < 4; i++) ss = fmaf(v[j].v[i], v[j].v[i], ss);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float inv = 1.0f / sqrtf(ss / (float)gs + n.eps);
  OutT *d = dst + (size_t)row * dst_stride + c0;
  const __nv_bfloat16 *w = n.w + (n.w_shared ? 0 : c0);
#pragma unroll
  for (int j = 0; j < MAXV; j++) {
    const int c = (lane + 32 * j) * 4;
    if (c < gs) {
      const FV<4> wv = ldw<4>(w + c);
#pragma unroll
      for (int i = 0; i < 4; i++) v[j].v[i] = v[j].v[i] * inv * wv.v[i];
      if (n.gate) gate_by(v[j], n.gate + (size_t)row * n.gate_stride + c0 + c);
      stv<4>(d + c, v[j]);
    }
  }
}

// short parts (at most 128 values): a warp takes four of them, so that enough loads are under way
template <typename OutT>
__global__ void __launch_bounds__(256) group_norm_short_kernel(const float *__restrict__ x, int x_stride, const GroupNorm n, int gs, OutT *__restrict__ dst,
                                                               int dst_stride, int rows) {
  pdl_launch();
  pdl_wait();
  constexpr int PARTS = 4;
  const int lane = threadIdx.x & 31, part0 = (blockIdx.x * 8 + (threadIdx.x >> 5)) * PARTS, c = lane * 4;
  FV<4> v[PARTS], gate[PARTS];
  int row[PARTS], at[PARTS];
#pragma unroll
  for (int i = 0; i < PARTS; i++) {
    const int part = part0 + i;
    row[i] = part / n.groups;
    at[i] = (part - row[i] * n.groups) * gs + c;
    const bool ok = part < rows * n.groups && c < gs;
    if (!ok) row[i] = -1;
    v[i] = ok ? ldv<4>(x + (size_t)row[i] * x_stride + at[i]) : FV<4>{};
    gate[i] = ok && n.gate ? ldv<4>(n.gate + (size_t)row[i] * n.gate_stride + at[i]) : FV<4>{};
  }
  float ss[PARTS];
#pragma unroll
  for (int i = 0; i < PARTS; i++) ss[i] = fmaf(v[i].v[0], v[i].v[0], fmaf(v[i].v[1], v[i].v[1], fmaf(v[i].v[2], v[i].v[2], v[i].v[3] * v[i].v[3])));
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int i = 0; i < PARTS; i++) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
#pragma unroll
  for (int i = 0; i < PARTS; i++) {
    if (row[i] < 0) continue;
    const float inv = 1.0f / sqrtf(ss[i] / (float)gs + n.eps);
    const FV<4> w = ldw<4>(n.w + (n.w_shared ? c : at[i]));
#pragma unroll
    for (int j = 0; j < 4; j++) {
      v[i].v[j] = v[i].v[j] * inv * w.v[j];
      if (n.gate) v[i].v[j] *= 1.0f / (1.0f + expf(-gate[i].v[j]));
    }
    stv<4>(dst + (size_t)row[i] * dst_stride + at[i], v[i]);
  }
}

template <int V, typename OutT>
__global__ void __launch_bounds__(256) group_norm_kernel(const float *__restrict__ x, int x_stride, const GroupNorm n, int gs, OutT *__restrict__ dst,
                                                         int dst_stride) {
  pdl_launch();
  pdl_wait();
  __shared__ float sh[8];
  const int c0 = blockIdx.y * gs, tid = threadIdx.x;
  const float *xr = x + (size_t)blockIdx.x * x_stride + c0;
  const FV<V> first = tid * V < gs ? ldv<V>(xr + tid * V) : FV<V>{};  // kept for the second pass
  float ss = 0.0f;
  for (int c = tid * V; c < gs; c += 256 * V) {
    const FV<V> v = c == tid * V ? first : ldv<V>(xr + c);
#pragma unroll
    for (int i = 0; i < V; i++) ss = fmaf(v.v[i], v.v[i], ss);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((tid & 31) == 0) sh[tid >> 5] = ss;
  __syncthreads();
  float t = 0.0f;
#pragma unroll
  for (int i = 0; i < 8; i++) t += sh[i];
  const float inv = 1.0f / sqrtf(t / (float)gs + n.eps);
  OutT *d = dst + (size_t)blockIdx.x * dst_stride + c0;
  const __nv_bfloat16 *w = n.w + (n.w_shared ? 0 : c0);
  for (int c = tid * V; c < gs; c += 256 * V) {
    FV<V> v = c == tid * V ? first : ldv<V>(xr + c);
    const FV<V> wv = ldw<V>(w + c);
#pragma unroll
    for (int i = 0; i < V; i++) v.v[i] = v.v[i] * inv * wv.v[i];
    if (n.gate) gate_by(v, n.gate + (size_t)blockIdx.x * n.gate_stride + c0 + c);
    stv<V>(d + c, v);
  }
}

__global__ void __launch_bounds__(256) hist_commit_kernel(const HistEntry *__restrict__ entries, int rows, int start_pos, int seq) {
  const HistEntry e = entries[blockIdx.y];
  const int n = min(rows, e.taps - 1);
  for (int c = blockIdx.x * 256 + threadIdx.x; c < e.channels; c += gridDim.x * 256)
    for (int k = 0; k < n; k++) {
      const size_t off = (size_t)((start_pos + rows - 1 - k) % e.taps) * e.channels + c;
      e.hist[(size_t)seq * e.hist_seq + off] = e.stage[off];
    }
}

unsigned flat_grid(dp_ctx *ctx, size_t n) {
  size_t g = (n + 255) / 256;
  const size_t cap = (size_t)ctx->sm_count * 16;
  return (unsigned)(g < cap ? (g ? g : 1) : cap);
}

}  // namespace

dp_status dpk_stream_boundary(dp_ctx *ctx, const float *x, float *x_out, const float *y, const SublayerOut &end, const SublayerIn &next, int streams, int width,
                              void *dst, bool dst_bf16, int dst_stride, int rows, const RowMap &map) {
  if (streams == 1 && next.groups == 1 && next.taps == 0 && end.groups == 1 && width % 4 == 0 && width <= 8192 && dst_stride % 4 == 0)
    return dst_bf16 ? launch_row(ctx, x, x_out, y, end, next, width, (__nv_bfloat16 *)dst, dst_stride, rows)
                    : launch_row(ctx, x, x_out, y, end, next, width, (float *)dst, dst_stride, rows);
  const int gs = width / next.groups;
  const int halo = (map.pos || next.taps < 2) ? 0 : next.taps - 1;
  const size_t row_bytes = (size_t)gs * 4;
  // Rows per CTA: the shape with the fewest rounds of the CTA's warps (reached-back rows included) on two CTAs per SM.
  const int cap = (int)(((size_t)ctx->smem_optin - 4096) / row_bytes), want = (int)((size_t)102400 / row_bytes);
  if (cap < 1 + halo) return dp_fail(ctx, DP_ERR_UNSUPPORTED, "streams: %d channels per norm group and %d taps exceed shared memory", gs, next.taps);
  int most = (want < cap ? want : cap) - halo;
  if (most < 1) most = 1;
  if (most > 32) most = 32;
  if (most > rows) most = rows;
  int R = 1;
  long best = -1;
  for (int r = 1; r <= most; r++) {
    const long blocks = (long)((rows + r - 1) / r) * next.groups, slots = 2l * ctx->sm_count;
    const long cost = ((blocks + slots - 1) / slots) * ((r + halo + SB_WARPS - 1) / SB_WARPS);
    if (best < 0 || cost < best) { best = cost; R = r; }
  }
  BoundaryArgs a;
  a.x = x; a.y = y; a.x_out = x_out; a.end = end; a.next = next;
  a.streams = streams; a.width = width; a.rows = rows; a.dst_stride = dst_stride; a.block_rows = R; a.map = map;
  const dim3 grid((rows + R - 1) / R, next.groups);
  const size_t smem = (size_t)(R + halo) * row_bytes;
  const bool vec = gs % 4 == 0 && dst_stride % 4 == 0;
  if (streams <= 4) return vec ? launch_boundary<4, 4>(ctx, a, dst, dst_bf16, grid, smem) : launch_boundary<4, 1>(ctx, a, dst, dst_bf16, grid, smem);
  return vec ? launch_boundary<DP_MAX_STREAMS, 4>(ctx, a, dst, dst_bf16, grid, smem) : launch_boundary<DP_MAX_STREAMS, 1>(ctx, a, dst, dst_bf16, grid, smem);
}

dp_status dpk_stream_sum(dp_ctx *ctx, const float *x, const float *y, const SublayerOut &end, int streams, int width, float *h, int rows) {
  if (end.norm_w && streams == 1 && end.groups == 1 && width % 4 == 0 && width <= 8192)
    return launch_row(ctx, x, h, y, end, SublayerIn(), width, (float *)nullptr, 0, rows);
  if (end.norm_w) {
    DP_LAUNCH(ctx, stream_sum_norm_kernel, rows, 256, 0, x, y, end, streams, width, h);
    return DP_OK;
  }
  DP_LAUNCH(ctx, stream_sum_kernel, flat_grid(ctx, (size_t)rows * width), 256, 0, x, y, end, streams, width, h, rows);
  return DP_OK;
}

dp_status dpk_stream_embed(dp_ctx *ctx, const int *ids, const __nv_bfloat16 *table, int table_stride, float scale, int streams, int width, float *x,
                           const float *in, float *u, int rows) {
  DP_LAUNCH(ctx, stream_embed_kernel, flat_grid(ctx, (size_t)rows * width), 256, 0, ids, table, table_stride, scale, streams, width, x, in, u, rows);
  return DP_OK;
}

dp_status dpk_group_norm(dp_ctx *ctx, const float *x, int x_stride, const GroupNorm &n, int width, void *dst, bool dst_bf16, int dst_stride, int rows) {
  const dim3 grid(rows, n.groups);
  const int gs = width / n.groups;
  const bool aligned = ((uintptr_t)x & 15) == 0 && (!n.gate || (((uintptr_t)n.gate & 15) == 0 && n.gate_stride % 4 == 0));
  const bool vec = gs % 4 == 0 && x_stride % 4 == 0 && dst_stride % 4 == 0 && aligned;
  if (vec && gs <= 128) {
    const unsigned blocks = (unsigned)(((size_t)rows * n.groups + 31) / 32);
    if (dst_bf16) DP_LAUNCH(ctx, group_norm_short_kernel<__nv_bfloat16>, blocks, 256, 0, x, x_stride, n, gs, (__nv_bfloat16 *)dst, dst_stride, rows);
    else DP_LAUNCH(ctx, group_norm_short_kernel<float>, blocks, 256, 0, x, x_stride, n, gs, (float *)dst, dst_stride, rows);
    return DP_OK;
  }
  if (vec && gs <= 1024) {
    const unsigned blocks = (unsigned)(((size_t)rows * n.groups + 7) / 8);
    if (dst_bf16) DP_LAUNCH(ctx, (group_norm_warp_kernel<8, __nv_bfloat16>), blocks, 256, 0, x, x_stride, n, gs, (__nv_bfloat16 *)dst, dst_stride, rows);
    else DP_LAUNCH(ctx, (group_norm_warp_kernel<8, float>), blocks, 256, 0, x, x_stride, n, gs, (float *)dst, dst_stride, rows);
    return DP_OK;
  }
#define DP_NORM(V, T) DP_LAUNCH(ctx, (group_norm_kernel<V, T>), grid, 256, 0, x, x_stride, n, gs, (T *)dst, dst_stride)
  if (dst_bf16) { if (vec) DP_NORM(4, __nv_bfloat16); else DP_NORM(1, __nv_bfloat16); }
  else { if (vec) DP_NORM(4, float); else DP_NORM(1, float); }
#undef DP_NORM
  return DP_OK;
}

dp_status dpk_hist_commit(dp_ctx *ctx, const HistEntry *entries, int n_entries, int max_channels, int rows, int start_pos, int seq) {
  if (n_entries == 0) return DP_OK;
  const dim3 grid((max_channels + 255) / 256, n_entries);
  DP_LAUNCH(ctx, hist_commit_kernel, grid, 256, 0, entries, rows, start_pos, seq);
  return DP_OK;
}
