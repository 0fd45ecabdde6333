// What comes between the q / k / v projections and the attention kernels of a decoder described layer by layer: per-head
// division by the root mean square (no weight), q to its own rows, k and v appended to the caches.  One warp per
// (row, head), any head sizes.
#include "layers.h"
#include "pdl.cuh"

namespace {

template <typename KT> __device__ __forceinline__ KT kv_cast(float v);
template <> __device__ __forceinline__ float kv_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __half kv_cast<__half>(float v) { return __float2half_rn(v); }

template <typename KT>
__global__ void __launch_bounds__(256) unit_qk_kv_kernel(const float *__restrict__ qkv, int qkv_stride, float *__restrict__ q_out, KT *__restrict__ kc,
                                                         KT *__restrict__ vc, int H, int G, int D, int V, int unit, float eps, size_t k_seq, size_t v_seq,
                                                         int rows, const RowMap map) {
  pdl_launch();
  pdl_wait();
  const int heads = H + 2 * G, lane = threadIdx.x & 31;
  const int gw = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (gw >= rows * heads) return;
  const int row = gw / heads, hd = gw - row * heads;
  const int pos = map.pos ? map.pos[row] : map.start_pos + row;
  const int seq = map.pos ? row : map.seq;
  const float *src = qkv + (size_t)row * qkv_stride;
  if (hd >= H + G) {
    const int g = hd - H - G;
    src += (size_t)(H + G) * D + (size_t)g * V;
    KT *dst = vc + (size_t)seq * v_seq + ((size_t)pos * G + g) * V;
    for (int d = lane; d < V; d += 32) dst[d] = kv_cast<KT>(src[d]);
    return;
  }
  src += (size_t)hd * D;
  float inv = 1.0f;
  if (unit) {
    float ss = 0.0f;
    for (int d = lane; d < D; d += 32) ss = fmaf(src[d], src[d], ss);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    inv = 1.0f / sqrtf(ss / (float)D + eps);
  }
  if (hd < H) {
    float *dst = q_out + ((size_t)row * H + hd) * D;
    for (int d = lane; d < D; d += 32) dst[d] = src[d] * inv;
  } else {
    KT *dst = kc + (size_t)seq * k_seq + ((size_t)pos * G + (hd - H)) * D;
    for (int d = lane; d < D; d += 32) dst[d] = kv_cast<KT>(src[d] * inv);
  }
}

}  // namespace

dp_status dpk_unit_qk_kv(dp_ctx *ctx, const float *qkv, int qkv_stride, float *q_out, void *kc, void *vc, bool kv_f32, int heads, int kv_heads, int dim,
                         int vdim, bool unit_rms, float eps, size_t k_seq, size_t v_seq, int rows, const RowMap &map) {
  const int warps = rows * (heads + 2 * kv_heads);
  const unsigned grid = (unsigned)((warps + 7) / 8);
  if (kv_f32)
    DP_LAUNCH(ctx, unit_qk_kv_kernel<float>, grid, 256, 0, qkv, qkv_stride, q_out, (float *)kc, (float *)vc, heads, kv_heads, dim, vdim, unit_rms ? 1 : 0, eps,
              k_seq, v_seq, rows, map);
  else
    DP_LAUNCH(ctx, unit_qk_kv_kernel<__half>, grid, 256, 0, qkv, qkv_stride, q_out, (__half *)kc, (__half *)vc, heads, kv_heads, dim, vdim, unit_rms ? 1 : 0,
              eps, k_seq, v_seq, rows, map);
  return DP_OK;
}
