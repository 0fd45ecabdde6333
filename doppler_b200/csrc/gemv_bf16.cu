// One-row products with bf16 weights: y = W x, x in f32, f32 accumulation (the single-token decode step of a decoder
// described layer by layer; serves both activation precisions, bf16 weights times f32 activations are exact in f32).
//
// HBM bound: 2 bytes per weight once.  One CTA per SM, 16 warps, a warp takes two rows at a time; a lane streams
// 16-byte pieces of both rows, four steps ahead.  The vector sits in shared memory as two planes (elements 0-3 and
// 4-7 of every eight), so that the 16-byte reads of a warp are conflict free.  What precedes the product in the layer
// is rebuilt by every CTA in its prologue and what follows is done by the warp that holds the sum, so a layer is a
// handful of kernels:
//   NORM     grouped RMSNorm of a row, then (where the sublayer has one) the causal input convolution over the
//            sequence's history; CTA 0 appends the row to the history.  The history is a ring of `taps` positions, so
//            the slot written is none of the slots read.
//   ATTN     merge of the split-K attention partials, times the per-head output gate
//   STREAMS  x_t <- sum_s mix[s][t] x_s + out[t] y for the warp's rows, and u = sum_t in[t] x_t of the next sublayer
//   GLU      gated activation of a gate row and its up row
// Before griddepcontrol.wait a warp asks for its first rows' weights in L2 (cp.async.bulk.prefetch), so the weight
// stream runs while the previous kernel drains and while the prologue works.
#include "layers.h"
#include "pdl.cuh"

#include <cfloat>

namespace {

constexpr int GB_THREADS = 512, GB_WARPS = GB_THREADS / 32;

__device__ __forceinline__ int gb_slot(int k, int plane) { return ((k >> 2) & 1) * plane + ((k >> 3) << 2) + (k & 3); }

__device__ __forceinline__ void gb_prefetch_l2(const void *p, uint32_t bytes) {
  asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(p), "r"(bytes) : "memory");
}

__device__ __forceinline__ float4 gb_ld4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ void gb_w4(const __nv_bfloat16 *p, float (&w)[4]) {  // p 8-byte aligned
  const uint2 r = __ldg(reinterpret_cast<const uint2 *>(p));
  w[0] = __uint_as_float(r.x << 16); w[1] = __uint_as_float(r.x & 0xffff0000u);
  w[2] = __uint_as_float(r.y << 16); w[3] = __uint_as_float(r.y & 0xffff0000u);
}

// x (in shared memory) = input convolution of the grouped RMSNorm of p.x.  Every warp owns whole groups or an equal
// part of one, so the scale of its channels is one number.
__device__ __forceinline__ void gb_prologue_norm(const GemvBf16 &p, float *sx, int plane, float *red) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int groups = p.norm.groups, gs = p.K / groups, taps = p.norm.taps;
  const int parts = groups >= GB_WARPS ? 1 : GB_WARPS / groups;
  const bool vec = (gs & 3) == 0;
  const int unit = vec ? 4 : 1;
  const int part_len = ((gs / unit + parts - 1) / parts) * unit;
  const int tasks = groups * parts;
  for (int base = 0; base < tasks; base += GB_WARPS) {
    const int task = base + warp;
    const int g = task / parts, c_lo = g * gs + (task - g * parts) * part_len, c_hi = min(c_lo + part_len, (g + 1) * gs);
    float ss = 0.0f;
    if (task < tasks) {
      if (vec) {
        for (int c = c_lo + lane * 4; c < c_hi; c += 128) {
          const float4 v = gb_ld4(p.x + c);
          *reinterpret_cast<float4 *>(sx + gb_slot(c, plane)) = v;
          ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
      } else {
        for (int c = c_lo + lane; c < c_hi; c += 32) {
          const float v = p.x[c];
          sx[gb_slot(c, plane)] = v;
          ss = fmaf(v, v, ss);
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    }
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    if (task < tasks) {
      float total = 0.0f;
      for (int i = 0; i < parts; i++) total += red[(warp / parts) * parts + i];
      const float inv = 1.0f / sqrtf(total / (float)gs + p.norm.eps);
      const int pos = taps > 0 ? *p.pos : 0;
      const bool keep = taps > 1 && blockIdx.x == 0;
      if (vec && taps <= 4) {
        for (int c = c_lo + lane * 4; c < c_hi; c += 128) {
          float4 v = *reinterpret_cast<float4 *>(sx + gb_slot(c, plane));
          float w[4];
          gb_w4(p.norm.norm_w + c, w);
          float h[4] = {v.x * inv * w[0], v.y * inv * w[1], v.z * inv * w[2], v.w * inv * w[3]};
          float o[4] = {h[0], h[1], h[2], h[3]};
          if (taps > 0) {
            float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            const __nv_bfloat16 *cw = p.norm.conv_w + (size_t)c * taps;
#pragma unroll
            for (int k = 3; k > 0; k--) {
              if (k < taps) {
                float4 past = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (pos - k >= 0) past = gb_ld4(p.norm.hist + (size_t)((pos - k) % taps) * p.K + c);
                const int j = taps - 1 - k;
                acc[0] = fmaf(__bfloat162float(cw[j]), past.x, acc[0]);
                acc[1] = fmaf(__bfloat162float(cw[taps + j]), past.y, acc[1]);
                acc[2] = fmaf(__bfloat162float(cw[2 * taps + j]), past.z, acc[2]);
                acc[3] = fmaf(__bfloat162float(cw[3 * taps + j]), past.w, acc[3]);
              }
            }
#pragma unroll
            for (int i = 0; i < 4; i++) o[i] = h[i] + fmaf(__bfloat162float(cw[i * taps + taps - 1]), h[i], acc[i]);
            if (keep) *reinterpret_cast<float4 *>(p.norm.hist + (size_t)(pos % taps) * p.K + c) = make_float4(h[0], h[1], h[2], h[3]);
          }
          *reinterpret_cast<float4 *>(sx + gb_slot(c, plane)) = make_float4(o[0], o[1], o[2], o[3]);
        }
      } else {
        for (int c = c_lo + lane * unit; c < c_hi; c += 32 * unit)
          for (int i = 0; i < unit; i++) {
            const float h = sx[gb_slot(c + i, plane)] * inv * __bfloat162float(p.norm.norm_w[c + i]);
            float o = h;
            if (taps > 0) {
              const __nv_bfloat16 *cw = p.norm.conv_w + (size_t)(c + i) * taps;
              float acc = 0.0f;
              for (int k = taps - 1; k > 0; k--)
                if (pos - k >= 0) acc = fmaf(__bfloat162float(cw[taps - 1 - k]), p.norm.hist[(size_t)((pos - k) % taps) * p.K + c + i], acc);
              o = h + fmaf(__bfloat162float(cw[taps - 1]), h, acc);
              if (keep) p.norm.hist[(size_t)(pos % taps) * p.K + c + i] = h;
            }
            sx[gb_slot(c + i, plane)] = o;
          }
      }
    }
    __syncthreads();  // red is reused
  }
}

// x = attention output of one row, merged from its split partials, times the head's gate
__device__ __forceinline__ void gb_prologue_attn(const GemvBf16 &p, float *sx, int plane, float *red) {
  (void)red;
  const int tid = threadIdx.x, V = p.vdim, S = p.splits;
  for (int e = tid; e < p.K; e += GB_THREADS) {
    const int h = e / V, d = e - h * V;
    const float *pp = p.x + (size_t)h * S * (V + 2);
    float mm = -FLT_MAX;
    for (int s = 0; s < S; s++) mm = fmaxf(mm, pp[s * (V + 2) + V]);
    float ll = 0.0f, acc = 0.0f;
#pragma unroll 4
    for (int s = 0; s < S; s++) {
      const float *ps = pp + s * (V + 2);
      const float c = ps[V] == -FLT_MAX ? 0.0f : exp2f(ps[V] - mm);
      ll = fmaf(ps[V + 1], c, ll);
      acc = fmaf(ps[d], c, acc);
    }
    float v = ll > 0.0f ? acc / ll : 0.0f;
    if (p.gate) v *= 1.0f / (1.0f + expf(-p.gate[h]));
    sx[gb_slot(e, plane)] = v;
  }
}

__device__ __forceinline__ void gb_dot8(const uint4 &w, const float4 &a, const float4 &b, float &acc) {
  acc = fmaf(__uint_as_float(w.x << 16), a.x, acc);
  acc = fmaf(__uint_as_float(w.x & 0xffff0000u), a.y, acc);
  acc = fmaf(__uint_as_float(w.y << 16), a.z, acc);
  acc = fmaf(__uint_as_float(w.y & 0xffff0000u), a.w, acc);
  acc = fmaf(__uint_as_float(w.z << 16), b.x, acc);
  acc = fmaf(__uint_as_float(w.z & 0xffff0000u), b.y, acc);
  acc = fmaf(__uint_as_float(w.w << 16), b.z, acc);
  acc = fmaf(__uint_as_float(w.w & 0xffff0000u), b.w, acc);
}

__device__ __forceinline__ uint4 gb_ldw(const uint4 *p) {
  uint4 r;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(r.x), "=r"(r.y), "=r"(r.z), "=r"(r.w) : "l"(p));
  return r;
}

template <int SRC, int DST>
__global__ void __launch_bounds__(GB_THREADS, 2) gemv_bf16_kernel(const GemvBf16 p) {
  pdl_launch();
  extern __shared__ __align__(16) float gb_sx[];
  __shared__ float red[GB_WARPS];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pieces = p.w_stride >> 3;      // 16-byte pieces per row
  const int plane = pieces * 4;            // floats per plane
  const int pairs = (p.N + 1) / 2;
  // pairs of rows dealt to the CTAs first, then to the warps: every SM streams the same share
  const int pair0 = (int)blockIdx.x + (int)gridDim.x * warp, step = (int)gridDim.x * GB_WARPS;
  auto row_a = [&](int pr) { return DST == GEMV_DST_GLU ? ((pr >> 3) * 16 + (pr & 7)) : 2 * pr; };
  auto row_b = [&](int pr) { return DST == GEMV_DST_GLU ? row_a(pr) + 8 : (2 * pr + 1 < p.N ? 2 * pr + 1 : 2 * pr); };
  {  // the weights are constant: ask for the first rows before the previous kernel has finished
    const uint32_t row_bytes = (uint32_t)p.w_stride * 2u;
    if (lane < 4) {
      const int pr = pair0 + (lane >> 1) * step;
      if (pr < pairs) gb_prefetch_l2(p.w + (size_t)((lane & 1) ? row_b(pr) : row_a(pr)) * p.w_stride, row_bytes);
    }
  }
  pdl_wait();
  for (int k = p.K + tid; k < pieces * 8; k += GB_THREADS) gb_sx[gb_slot(k, plane)] = 0.0f;  // the padded tail
  if constexpr (SRC == GEMV_SRC_NORM) {
    gb_prologue_norm(p, gb_sx, plane, red);
  } else if constexpr (SRC == GEMV_SRC_ATTN) {
    gb_prologue_attn(p, gb_sx, plane, red);
  } else {
    for (int k = tid; k < p.K; k += GB_THREADS) gb_sx[gb_slot(k, plane)] = p.x[k];
  }
  __syncthreads();

  const float4 *x0 = reinterpret_cast<const float4 *>(gb_sx), *x1 = reinterpret_cast<const float4 *>(gb_sx + plane);
  for (int pr = pair0; pr < pairs; pr += step) {
    const int ra = row_a(pr), rb = row_b(pr);
    const uint4 *wa = reinterpret_cast<const uint4 *>(p.w + (size_t)ra * p.w_stride);
    const uint4 *wb = reinterpret_cast<const uint4 *>(p.w + (size_t)rb * p.w_stride);
    float a0 = 0.0f, b0 = 0.0f;
    int k = lane;
    for (; k + 96 < pieces; k += 128) {
      uint4 va[4], vb[4];
#pragma unroll
      for (int i = 0; i < 4; i++) { va[i] = gb_ldw(wa + k + 32 * i); vb[i] = gb_ldw(wb + k + 32 * i); }
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const float4 xa = x0[k + 32 * i], xb = x1[k + 32 * i];
        gb_dot8(va[i], xa, xb, a0);
        gb_dot8(vb[i], xa, xb, b0);
      }
    }
    for (; k < pieces; k += 32) {
      const uint4 va = gb_ldw(wa + k), vb = gb_ldw(wb + k);
      const float4 xa = x0[k], xb = x1[k];
      gb_dot8(va, xa, xb, a0);
      gb_dot8(vb, xa, xb, b0);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      a0 += __shfl_xor_sync(0xffffffffu, a0, o);
      b0 += __shfl_xor_sync(0xffffffffu, b0, o);
    }
    if constexpr (DST == GEMV_DST_PLAIN) {
      if (lane == 0) p.y[ra] = a0;
      if (lane == 1 && rb != ra) p.y[rb] = b0;
    } else if constexpr (DST == GEMV_DST_GLU) {
      if (lane == 0) {
        const float g = p.limit > 0.0f ? fminf(a0, p.limit) : a0;
        const float u = p.limit > 0.0f ? fminf(fmaxf(b0, -p.limit), p.limit) : b0;
        p.y[pr] = g * (1.0f / (1.0f + expf(-p.slope * g))) * (u + p.shift);
      }
    } else {
      // lane t < streams: stream t of row ra; lane 16 + t: of row rb
      const int t = lane & 15, r = lane < 16 ? ra : rb;
      const bool mine = t < p.streams && (lane < 16 || rb != ra);
      const float y = lane < 16 ? a0 : b0;
      float nx = 0.0f, part = 0.0f;
      if (mine) {
        nx = p.end.out[t] * y;
        for (int s = 0; s < p.streams; s++) nx = fmaf(p.end.mix[s * p.streams + t], p.streams_x[(size_t)s * p.N + r], nx);
        part = (p.next_in ? p.next_in[t] : 1.0f) * nx;
      }
      __syncwarp();  // every old value of the row has been read
      if (mine) p.streams_x[(size_t)t * p.N + r] = nx;
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) part += __shfl_xor_sync(0xffffffffu, part, o);
      if (t == 0 && (lane < 16 || rb != ra)) p.next_u[r] = part;
    }
  }
}

template <int SRC, int DST>
dp_status launch(dp_ctx *ctx, const GemvBf16 &p) {
  const size_t smem = (size_t)(p.w_stride) * 4;
  if (smem > ctx->smem_optin - 1024)
    return dp_fail(ctx, DP_ERR_UNSUPPORTED, "gemv (bf16): a vector of %d values exceeds shared memory", p.K);
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    DP_CUDA(ctx, cudaFuncSetAttribute((gemv_bf16_kernel<SRC, DST>), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ctx->smem_optin - 1024));
    attr.done(ctx->device);
  }
  const int pairs = (p.N + 1) / 2;
  const int grid = pairs < ctx->sm_count ? pairs : ctx->sm_count;
  DP_LAUNCH(ctx, (gemv_bf16_kernel<SRC, DST>), grid, GB_THREADS, smem, p);
  return DP_OK;
}

}  // namespace

dp_status dpk_gemv_bf16(dp_ctx *ctx, int src, int dst, const GemvBf16 &p) {
  if (p.w_stride % 8 || p.K > p.w_stride || p.streams > DP_MAX_STREAMS) return dp_fail(ctx, DP_ERR_INVALID, "gemv (bf16): bad row stride %d for K %d", p.w_stride, p.K);
  if (src == GEMV_SRC_PLAIN && dst == GEMV_DST_PLAIN) return launch<GEMV_SRC_PLAIN, GEMV_DST_PLAIN>(ctx, p);
  if (src == GEMV_SRC_PLAIN && dst == GEMV_DST_STREAMS) return launch<GEMV_SRC_PLAIN, GEMV_DST_STREAMS>(ctx, p);
  if (src == GEMV_SRC_NORM && dst == GEMV_DST_PLAIN) return launch<GEMV_SRC_NORM, GEMV_DST_PLAIN>(ctx, p);
  if (src == GEMV_SRC_NORM && dst == GEMV_DST_GLU) return launch<GEMV_SRC_NORM, GEMV_DST_GLU>(ctx, p);
  if (src == GEMV_SRC_NORM && dst == GEMV_DST_STREAMS) return launch<GEMV_SRC_NORM, GEMV_DST_STREAMS>(ctx, p);
  if (src == GEMV_SRC_ATTN && dst == GEMV_DST_STREAMS) return launch<GEMV_SRC_ATTN, GEMV_DST_STREAMS>(ctx, p);
  return dp_fail(ctx, DP_ERR_UNSUPPORTED, "gemv (bf16): no kernel for source %d and destination %d", src, dst);
}
