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
//   RESIDUAL x + out norm(y) of the sublayer that ended (y has a norm of its own, one stream), then NORM; CTA 0 stores the
//            sum to another buffer than the one that is read
//   GATED    NORM (its weight may serve every group), times the sigmoid of a gate per value
//   ATTN     merge of the split-K attention partials, times the per-head output gate
//   STREAMS  x_t <- sum_s mix[s][t] x_s + out[t] y for the warp's rows, and u = sum_t in[t] x_t of the next sublayer
//   GLU      gated activation of a gate row and its up row
// Before griddepcontrol.wait a warp asks for the start of its first rows in L2 (cp.async.bulk.prefetch) and the part of
// the input convolution that lies in the past is summed up, so both run while the previous kernel drains.
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

// The part of the input convolution that does not depend on this token: past[c] = sum over the history, and the two
// per-channel factors packed as a bf16 pair (norm weight, the convolution's last tap).  The history was written by
// earlier steps, so this runs before griddepcontrol.wait.
__device__ __forceinline__ void gb_conv_past(const GemvBf16 &p, float *past, uint32_t *fac) {
  const int taps = p.norm.taps, K = p.K, pos = *p.pos;
  const uint16_t *nw = reinterpret_cast<const uint16_t *>(p.norm.norm_w), *cw = reinterpret_cast<const uint16_t *>(p.norm.conv_w);
  if ((K & 3) == 0 && taps == 4) {
    const float *h1 = p.norm.hist + (size_t)((pos + 3) & 3) * K, *h2 = p.norm.hist + (size_t)((pos + 2) & 3) * K, *h3 = p.norm.hist + (size_t)((pos + 1) & 3) * K;
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 2
    for (int c = threadIdx.x * 4; c < K; c += GB_THREADS * 4) {
      const float4 a1 = pos >= 1 ? gb_ld4(h1 + c) : zero, a2 = pos >= 2 ? gb_ld4(h2 + c) : zero, a3 = pos >= 3 ? gb_ld4(h3 + c) : zero;
      const uint4 w01 = __ldg(reinterpret_cast<const uint4 *>(cw + (size_t)c * 4)), w23 = __ldg(reinterpret_cast<const uint4 *>(cw + (size_t)c * 4) + 1);
      const uint2 n = __ldg(reinterpret_cast<const uint2 *>(nw + c));
      const float q1[4] = {a1.x, a1.y, a1.z, a1.w}, q2[4] = {a2.x, a2.y, a2.z, a2.w}, q3[4] = {a3.x, a3.y, a3.z, a3.w};
      const uint32_t lo[4] = {w01.x, w01.z, w23.x, w23.z}, hi[4] = {w01.y, w01.w, w23.y, w23.w};  // taps 0, 1 and taps 2, 3 of a channel
      const uint32_t nn[4] = {n.x & 0xffffu, n.x >> 16, n.y & 0xffffu, n.y >> 16};
#pragma unroll
      for (int i = 0; i < 4; i++) {
        past[c + i] = fmaf(__uint_as_float(hi[i] << 16), q1[i], fmaf(__uint_as_float(lo[i] & 0xffff0000u), q2[i], __uint_as_float(lo[i] << 16) * q3[i]));
        fac[c + i] = nn[i] | (hi[i] & 0xffff0000u);
      }
    }
    return;
  }
  for (int c = threadIdx.x; c < K; c += GB_THREADS) {
    float acc = 0.0f;
    for (int k = taps - 1; k > 0; k--)
      if (pos - k >= 0) acc = fmaf(__bfloat162float(p.norm.conv_w[(size_t)c * taps + taps - 1 - k]), p.norm.hist[(size_t)((pos - k) % taps) * K + c], acc);
    past[c] = acc;
    fac[c] = (uint32_t)nw[c] | (uint32_t)cw[(size_t)c * taps + taps - 1] << 16;
  }
}

// x (in shared memory) = input convolution of the grouped RMSNorm of p.x.  Every warp owns whole groups or an equal
// part of one, so the scale of its channels is one number.
template <int SRC>
__device__ __forceinline__ void gb_prologue_norm(const GemvBf16 &p, float *sx, int plane, float *red, const float *past, const uint32_t *fac) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int groups = p.norm.groups, gs = p.K / groups, taps = p.norm.taps;
  const int parts = groups >= GB_WARPS ? 1 : GB_WARPS / groups;
  const bool vec = (gs & 3) == 0;
  const int unit = vec ? 4 : 1;
  const int part_len = ((gs / unit + parts - 1) / parts) * unit;
  const int tasks = groups * parts;
  const bool keep = taps > 1 && blockIdx.x == 0;
  const bool gate4 = SRC == GEMV_SRC_GATED && ((uintptr_t)p.gate & 15) == 0;
  float *slot = keep ? p.norm.hist + (size_t)(*p.pos % taps) * p.K : nullptr;
  for (int base = 0; base < tasks; base += GB_WARPS) {
    const int task = base + warp;
    const int g = task / parts, c_lo = g * gs + (task - g * parts) * part_len, c_hi = min(c_lo + part_len, (g + 1) * gs);
    float ss = 0.0f;
    if constexpr (SRC == GEMV_SRC_RESIDUAL) {
      // the sum, into shared memory; res.groups equals groups
      float sy = 0.0f;
      if (task < tasks) {
        if (vec) {
#pragma unroll 4
          for (int c = c_lo + lane * 4; c < c_hi; c += 128) {
            const float4 v = gb_ld4(p.res_y + c);
            *reinterpret_cast<float4 *>(sx + gb_slot(c, plane)) = v;
            sy = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, sy))));
          }
        } else {
          for (int c = c_lo + lane; c < c_hi; c += 32) {
            const float v = p.res_y[c];
            sx[gb_slot(c, plane)] = v;
            sy = fmaf(v, v, sy);
          }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sy += __shfl_xor_sync(0xffffffffu, sy, o);
      }
      if (lane == 0) red[GB_WARPS + warp] = sy;
      __syncthreads();
      if (task < tasks) {
        float total = 0.0f;
        for (int i = 0; i < parts; i++) total += red[GB_WARPS + (warp / parts) * parts + i];
        const float f = p.res.out[0] / sqrtf(total / (float)gs + p.res.eps);
        const float mix = p.res.mix[0];
        if (vec) {
#pragma unroll 4
          for (int c = c_lo + lane * 4; c < c_hi; c += 128) {
            float4 *slot4 = reinterpret_cast<float4 *>(sx + gb_slot(c, plane));
            const float4 y = *slot4, x = gb_ld4(p.x + c);
            float w[4];
            gb_w4(p.res.norm_w + c, w);
            const float4 v = make_float4(fmaf(mix, x.x, f * y.x * w[0]), fmaf(mix, x.y, f * y.y * w[1]), fmaf(mix, x.z, f * y.z * w[2]), fmaf(mix, x.w, f * y.w * w[3]));
            *slot4 = v;
            if (blockIdx.x == 0) *reinterpret_cast<float4 *>(p.x_out + c) = v;
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
          }
        } else {
          for (int c = c_lo + lane; c < c_hi; c += 32) {
            const float v = fmaf(mix, p.x[c], f * sx[gb_slot(c, plane)] * __bfloat162float(p.res.norm_w[c]));
            sx[gb_slot(c, plane)] = v;
            if (blockIdx.x == 0) p.x_out[c] = v;
            ss = fmaf(v, v, ss);
          }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      }
    } else if (task < tasks) {
      if (vec) {
#pragma unroll 4
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
      for (int c = c_lo + lane * unit; c < c_hi; c += 32 * unit) {
        float v[4], w[4];
        if (vec) {
          const float4 q = *reinterpret_cast<float4 *>(sx + gb_slot(c, plane));
          v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
        } else v[0] = sx[gb_slot(c, plane)];
        if (taps > 0) {
#pragma unroll
          for (int i = 0; i < 4; i++)
            if (i < unit) {
              const uint32_t f = fac[c + i];
              const float h = v[i] * inv * __uint_as_float(f << 16);
              if (keep) slot[c + i] = h;
              v[i] = h + fmaf(__uint_as_float(f & 0xffff0000u), h, past[c + i]);
            }
        } else {
          const __nv_bfloat16 *nw = p.norm.norm_w + (SRC == GEMV_SRC_GATED && p.norm_w_shared ? c - g * gs : c);
          if (vec) {
            gb_w4(nw, w);
#pragma unroll
            for (int i = 0; i < 4; i++) v[i] = v[i] * inv * w[i];
          } else v[0] = v[0] * inv * __bfloat162float(*nw);
        }
        if constexpr (SRC == GEMV_SRC_GATED) {
          if (vec && gate4) {
            const float4 q = gb_ld4(p.gate + c);
            v[0] *= 1.0f / (1.0f + expf(-q.x)); v[1] *= 1.0f / (1.0f + expf(-q.y));
            v[2] *= 1.0f / (1.0f + expf(-q.z)); v[3] *= 1.0f / (1.0f + expf(-q.w));
          } else {
#pragma unroll
            for (int i = 0; i < 4; i++)
              if (i < unit) v[i] *= 1.0f / (1.0f + expf(-p.gate[c + i]));
          }
        }
        if (vec) *reinterpret_cast<float4 *>(sx + gb_slot(c, plane)) = make_float4(v[0], v[1], v[2], v[3]);
        else sx[gb_slot(c, plane)] = v[0];
      }
    }
    if (base + GB_WARPS < tasks) __syncthreads();  // red is reused
  }
}

// x = attention output of one row, merged from its split partials, times the head's gate.  wgt [head][split]: what a
// split's partial counts for.
__device__ __forceinline__ void gb_prologue_attn(const GemvBf16 &p, float *sx, int plane, float *wgt) {
  const int tid = threadIdx.x, lane = tid & 31, V = p.vdim, S = p.splits, row = V + 2;
  for (int h = tid >> 5; h < p.heads; h += GB_WARPS) {  // a warp per head, a lane per split (at most 32)
    const float *pp = p.x + ((size_t)h * S + lane) * row + V;
    const float m = lane < S ? pp[0] : -FLT_MAX, l = lane < S ? pp[1] : 0.0f;
    const float g = p.gate ? p.gate[h] : 0.0f;
    float mm = m;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffffu, mm, o));
    const float c = m == -FLT_MAX ? 0.0f : exp2f(m - mm);
    float ll = l * c;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ll += __shfl_xor_sync(0xffffffffu, ll, o);
    float f = ll > 0.0f ? c / ll : 0.0f;
    if (p.gate) f *= 1.0f / (1.0f + expf(-g));
    if (lane < S) wgt[h * S + lane] = f;
  }
  __syncthreads();
  if ((V & 1) == 0) {
#pragma unroll 2
    for (int e = 2 * tid; e < p.K; e += 2 * GB_THREADS) {
      const int h = e / V;
      const float *pp = p.x + (size_t)h * S * row + (e - h * V), *wh = wgt + h * S;
      float a0 = 0.0f, a1 = 0.0f;
#pragma unroll 8
      for (int s = 0; s < S; s++) {
        const float2 v = *reinterpret_cast<const float2 *>(pp + s * row);
        a0 = fmaf(v.x, wh[s], a0);
        a1 = fmaf(v.y, wh[s], a1);
      }
      *reinterpret_cast<float2 *>(sx + gb_slot(e, plane)) = make_float2(a0, a1);
    }
  } else {
    for (int e = tid; e < p.K; e += GB_THREADS) {
      const int h = e / V;
      const float *pp = p.x + (size_t)h * S * row + (e - h * V), *wh = wgt + h * S;
      float acc = 0.0f;
      for (int s = 0; s < S; s++) acc = fmaf(pp[s * row], wh[s], acc);
      sx[gb_slot(e, plane)] = acc;
    }
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
  extern __shared__ __align__(16) float gb_sx[];
  __shared__ float red[2 * GB_WARPS];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pieces = p.w_stride >> 3;      // 16-byte pieces per row
  const int plane = pieces * 4;            // floats per plane
  const int pairs = (p.N + 1) / 2;
  // pairs of rows dealt to the CTAs first, then to the warps: every SM streams the same share
  const int pair0 = (int)blockIdx.x + (int)gridDim.x * warp, step = (int)gridDim.x * GB_WARPS;
  auto row_a = [&](int pr) { return DST == GEMV_DST_GLU ? ((pr >> 3) * 16 + (pr & 7)) : 2 * pr; };
  auto row_b = [&](int pr) { return DST == GEMV_DST_GLU ? row_a(pr) + 8 : (2 * pr + 1 < p.N ? 2 * pr + 1 : 2 * pr); };
  float *extra = gb_sx + 2 * plane;  // behind the vector: what the prologue needs beside it
  {  // the weights are constant: ask for the start of the first rows before the previous kernel has finished
    const uint32_t row_bytes = min((uint32_t)p.w_stride * 2u, p.prefetch_bytes);
    if (lane < 2 && pair0 < pairs && row_bytes) gb_prefetch_l2(p.w + (size_t)(lane ? row_b(pair0) : row_a(pair0)) * p.w_stride, row_bytes);
  }
  for (int k = p.K + tid; k < pieces * 8; k += GB_THREADS) gb_sx[gb_slot(k, plane)] = 0.0f;  // the padded tail
  constexpr bool NORMS = SRC == GEMV_SRC_NORM || SRC == GEMV_SRC_RESIDUAL || SRC == GEMV_SRC_GATED;
  if constexpr (NORMS)
    if (p.norm.taps > 0) gb_conv_past(p, extra, reinterpret_cast<uint32_t *>(extra) + p.K);
  pdl_wait();
  pdl_launch();  // not before the wait: the next kernel's early work then competes with this kernel's stream only
  if constexpr (NORMS) {
    if (p.norm.taps > 0) __syncthreads();
    gb_prologue_norm<SRC>(p, gb_sx, plane, red, extra, reinterpret_cast<const uint32_t *>(extra) + p.K);
  } else if constexpr (SRC == GEMV_SRC_ATTN) {
    gb_prologue_attn(p, gb_sx, plane, extra);
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
  size_t smem = (size_t)p.w_stride * 4;
  if (SRC != GEMV_SRC_PLAIN && SRC != GEMV_SRC_ATTN && p.norm.taps > 0) smem += (size_t)p.K * 8;
  if (SRC == GEMV_SRC_ATTN) smem += (size_t)p.heads * p.splits * 4;
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
  if (src == GEMV_SRC_ATTN && dst == GEMV_DST_PLAIN) return launch<GEMV_SRC_ATTN, GEMV_DST_PLAIN>(ctx, p);
  if (src == GEMV_SRC_RESIDUAL && dst == GEMV_DST_PLAIN) return launch<GEMV_SRC_RESIDUAL, GEMV_DST_PLAIN>(ctx, p);
  if (src == GEMV_SRC_RESIDUAL && dst == GEMV_DST_GLU) return launch<GEMV_SRC_RESIDUAL, GEMV_DST_GLU>(ctx, p);
  if (src == GEMV_SRC_GATED && dst == GEMV_DST_PLAIN) return launch<GEMV_SRC_GATED, GEMV_DST_PLAIN>(ctx, p);
  return dp_fail(ctx, DP_ERR_UNSUPPORTED, "gemv (bf16): no kernel for source %d and destination %d", src, dst);
}
