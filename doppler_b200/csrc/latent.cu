// Latent attention: what happens around the attention kernels.
//
// The cache of a layer holds one row per token, [c | rotated key part] (see LatentShape), from which keys and values of all
// heads follow: k_h = W_uk,h c, v_h = W_uv,h c.  A query meets the cache in one of two ways:
//   absorbed   q_h . (W_uk,h c) = (W_uk,h^T q_h) . c, so the queries are brought into the latent space once and the attention
//              runs on the cache rows themselves, which all heads share; its result is a mean of c, and W_uv,h turns it into
//              values.  Decode steps, short portions and the 32-bit mode.
//   expanded   keys and values of all cached tokens are formed by one product and the attention runs on those: fewer
//              operations per (query, key), worth it for portions of many rows.
#include "layers.h"
#include "pdl.cuh"

#include <cfloat>

namespace {

template <typename KT> __device__ __forceinline__ KT lt_cast(float v);
template <> __device__ __forceinline__ float lt_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __half lt_cast<__half>(float v) { return __float2half_rn(v); }

__device__ __forceinline__ float lt_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }

// sum over a CTA of 256 threads
__device__ __forceinline__ float lt_block_sum(float v, float *red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.0f;
#pragma unroll
  for (int i = 0; i < 8; i++) t += red[i];
  return t;
}

// a token's cache row from its projections (256 threads)
template <typename KT>
__device__ __forceinline__ void lt_append_row(const float *dkv, const LatentShape &sh, const __nv_bfloat16 *norm_w, const Rotation &rot, KT *row, int pos, float *red) {
  const int tid = threadIdx.x, half = sh.rot_dim / 2;
  float ss = 0.0f;
  for (int c = tid; c < sh.kv_rank; c += 256) ss = fmaf(dkv[c], dkv[c], ss);
  const float inv = 1.0f / sqrtf(lt_block_sum(ss, red) / (float)sh.kv_rank + sh.eps);
  for (int c = tid; c < sh.kv_rank; c += 256) row[c] = lt_cast<KT>(dkv[c] * inv * __bfloat162float(norm_w[c]));
  for (int i = tid; i < half; i += 256) {
    const float co = rot.cos_t[(size_t)pos * half + i], si = rot.sin_t[(size_t)pos * half + i];
    const float u = dkv[sh.kv_rank + i], v = dkv[sh.kv_rank + half + i];
    row[sh.c_pad() + i] = lt_cast<KT>(u * co - v * si);
    row[sh.c_pad() + half + i] = lt_cast<KT>(v * co + u * si);
  }
}

// pair i of a head's rotated query part, in place or to the tail of its absorbed row
__device__ __forceinline__ void lt_rotate_query(float *q, float *q_abs, const LatentShape &sh, const Rotation &rot, int pos, int i) {
  const int half = sh.rot_dim / 2;
  const float co = rot.cos_t[(size_t)pos * half + i], si = rot.sin_t[(size_t)pos * half + i];
  const float u = q[sh.dim + i], v = q[sh.dim + half + i];
  float *dst = q_abs ? q_abs + sh.c_pad() : q + sh.dim;
  dst[i] = u * co - v * si;
  dst[half + i] = v * co + u * si;
}
// the zeros between and behind the parts of an absorbed query row
__device__ __forceinline__ void lt_query_pads(float *q_abs, const LatentShape &sh, int i, int step) {
  for (int c = sh.kv_rank + i; c < sh.c_pad(); c += step) q_abs[c] = 0.0f;
  for (int c = sh.c_pad() + sh.rot_dim + i; c < sh.cols(); c += step) q_abs[c] = 0.0f;
}

template <typename KT>
__global__ void __launch_bounds__(256) latent_append_kernel(const float *__restrict__ proj, int proj_stride, const LatentShape sh,
                                                            const __nv_bfloat16 *__restrict__ norm_w, const Rotation rot, const LatentCache cache, float *q, float *q_rot,
                                                            const RowMap map) {
  pdl_launch();
  pdl_wait();
  __shared__ float red[8];
  const int row = blockIdx.x, half = sh.rot_dim / 2;
  const int pos = map.pos ? map.pos[row] : map.start_pos + row, seq = map.pos ? row : map.seq;
  lt_append_row<KT>(proj + (size_t)row * proj_stride + sh.dkv_col(), sh, norm_w, rot, (KT *)cache.rows + (size_t)seq * cache.seq + (size_t)pos * sh.cols(), pos, red);
  for (int i = threadIdx.x; i < sh.heads * half; i += 256) {
    const int h = i / half;
    const size_t hr = (size_t)row * sh.heads + h;
    lt_rotate_query(q + hr * (sh.dim + sh.rot_dim), q_rot ? q_rot + hr * sh.cols() : nullptr, sh, rot, pos, i - h * half);
  }
  if (q_rot)
    for (int h = threadIdx.x; h < sh.heads; h += 256) lt_query_pads(q_rot + ((size_t)row * sh.heads + h) * sh.cols(), sh, 0, 1);
}

// ---- one decode row: grid (heads + 1, tiles of 128 latent channels); the blocks behind the heads append the cache row ----
// A thread owns eight channels and every sixteenth key dimension; its first weights are asked for before the wait.
constexpr int LA_COLS = 128, LA_PRE = 8;
template <typename KT>
__global__ void __launch_bounds__(256) latent_absorb_step_kernel(const float *__restrict__ proj, const LatentShape sh, const __nv_bfloat16 *__restrict__ norm_w,
                                                                 const Rotation rot, const LatentCache cache, const __nv_bfloat16 *__restrict__ wuk, int wuk_stride,
                                                                 const float *__restrict__ q, float *__restrict__ q_abs, const int *__restrict__ pos_arr) {
  __shared__ __align__(16) float part[16][LA_COLS + 4];
  __shared__ float red[8];
  const int tid = threadIdx.x, h = blockIdx.x, half = sh.rot_dim / 2, pos = pos_arr[0];
  if (h == sh.heads) {
    pdl_wait();
    pdl_launch();
    if (blockIdx.y == 0) lt_append_row<KT>(proj + sh.dkv_col(), sh, norm_w, rot, (KT *)cache.rows + (size_t)pos * sh.cols(), pos, red);
    return;
  }
  const int dg = tid >> 4, c0 = blockIdx.y * LA_COLS + (tid & 15) * 8;
  const bool mine = c0 < wuk_stride;
  const __nv_bfloat16 *w = wuk + (size_t)h * sh.dim * wuk_stride + c0;
  uint4 pre[LA_PRE];
#pragma unroll
  for (int i = 0; i < LA_PRE; i++) {
    const int d = dg + 16 * i;
    pre[i] = mine && d < sh.dim ? __ldg(reinterpret_cast<const uint4 *>(w + (size_t)d * wuk_stride)) : make_uint4(0, 0, 0, 0);
  }
  pdl_wait();
  pdl_launch();
  const float *qh = q + (size_t)h * (sh.dim + sh.rot_dim);
  float acc[8] = {};
  auto add = [&](const uint4 &v, float x) {
    acc[0] = fmaf(__uint_as_float(v.x << 16), x, acc[0]); acc[1] = fmaf(__uint_as_float(v.x & 0xffff0000u), x, acc[1]);
    acc[2] = fmaf(__uint_as_float(v.y << 16), x, acc[2]); acc[3] = fmaf(__uint_as_float(v.y & 0xffff0000u), x, acc[3]);
    acc[4] = fmaf(__uint_as_float(v.z << 16), x, acc[4]); acc[5] = fmaf(__uint_as_float(v.z & 0xffff0000u), x, acc[5]);
    acc[6] = fmaf(__uint_as_float(v.w << 16), x, acc[6]); acc[7] = fmaf(__uint_as_float(v.w & 0xffff0000u), x, acc[7]);
  };
#pragma unroll
  for (int i = 0; i < LA_PRE; i++) {
    const int d = dg + 16 * i;
    if (d < sh.dim) add(pre[i], qh[d]);
  }
  if (mine)
    for (int d = dg + 16 * LA_PRE; d < sh.dim; d += 16) add(__ldg(reinterpret_cast<const uint4 *>(w + (size_t)d * wuk_stride)), qh[d]);
  float *dst = part[dg] + (tid & 15) * 8;
  *reinterpret_cast<float4 *>(dst) = make_float4(acc[0], acc[1], acc[2], acc[3]);
  *reinterpret_cast<float4 *>(dst + 4) = make_float4(acc[4], acc[5], acc[6], acc[7]);
  __syncthreads();
  float *out = q_abs + (size_t)h * sh.cols();
  if (tid < LA_COLS) {
    const int c = blockIdx.y * LA_COLS + tid;
    float v = 0.0f;
#pragma unroll
    for (int i = 0; i < 16; i++) v += part[i][tid];
    if (c < sh.kv_rank) out[c] = v;
  } else if (blockIdx.y == 0) {
    for (int i = tid - LA_COLS; i < half; i += 256 - LA_COLS) lt_rotate_query(const_cast<float *>(qh), out, sh, rot, pos, i);
    lt_query_pads(out, sh, tid - LA_COLS, 256 - LA_COLS);
  }
}

// ---- one decode row: merge of the split partials and the value matrix, grid (heads, tiles of 32 values) ----
constexpr int LV_ROWS = 32;
__global__ void __launch_bounds__(256) latent_values_step_kernel(const float *__restrict__ part, int splits, const LatentShape sh, const __nv_bfloat16 *__restrict__ wuv,
                                                                 int wuv_stride, const float *__restrict__ gate, float *__restrict__ out) {
  extern __shared__ __align__(16) float lv_ctx[];  // [wuv_stride]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, v0 = blockIdx.y * LV_ROWS;
  const int pieces = wuv_stride / 8, CP = sh.c_pad(), row = CP + 2;
  constexpr int PER = LV_ROWS / 8, PRE = 2;  // rows per warp, pieces asked for before the wait
  uint4 pre[PER][PRE];
#pragma unroll
  for (int i = 0; i < PER; i++) {
    const int v = v0 + warp * PER + i;
    const uint4 *w = reinterpret_cast<const uint4 *>(wuv + ((size_t)h * sh.vdim + v) * wuv_stride);
#pragma unroll
    for (int j = 0; j < PRE; j++) pre[i][j] = v < sh.vdim && lane + 32 * j < pieces ? __ldg(w + lane + 32 * j) : make_uint4(0, 0, 0, 0);
  }
  pdl_wait();
  pdl_launch();
  const float *pp = part + (size_t)h * splits * (splits > 1 ? row : CP);
  if (splits > 1) {
    // every warp works out what each split counts for, a lane per split
    const float m = lane < splits ? pp[(size_t)lane * row + CP] : -FLT_MAX, l = lane < splits ? pp[(size_t)lane * row + CP + 1] : 0.0f;
    float mm = m;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffffu, mm, o));
    const float c = m == -FLT_MAX ? 0.0f : exp2f(m - mm);
    float ll = l * c;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ll += __shfl_xor_sync(0xffffffffu, ll, o);
    const float wt = ll > 0.0f ? c / ll : 0.0f;
    for (int c0 = 0; c0 < CP; c0 += 512) {  // two columns per thread, c_pad is a multiple of sixteen
      const int k = c0 + 2 * tid;
      float2 acc = make_float2(0.0f, 0.0f);
#pragma unroll 16
      for (int s = 0; s < splits; s++) {
        const float f = __shfl_sync(0xffffffffu, wt, s);
        const float2 x = k < CP ? *reinterpret_cast<const float2 *>(pp + (size_t)s * row + k) : make_float2(0.0f, 0.0f);
        acc.x = fmaf(x.x, f, acc.x);
        acc.y = fmaf(x.y, f, acc.y);
      }
      if (k < wuv_stride) *reinterpret_cast<float2 *>(lv_ctx + k) = acc;
    }
  } else {
    for (int c = tid; c < wuv_stride; c += 256) lv_ctx[c] = pp[c];
  }
  __syncthreads();
  const float g = gate ? lt_sigmoid(gate[h]) : 1.0f;
  auto dot = [&](const uint4 &r, int k, float acc) {
    const float4 a = *reinterpret_cast<const float4 *>(lv_ctx + 8 * k), b = *reinterpret_cast<const float4 *>(lv_ctx + 8 * k + 4);
    acc = fmaf(__uint_as_float(r.x << 16), a.x, acc); acc = fmaf(__uint_as_float(r.x & 0xffff0000u), a.y, acc);
    acc = fmaf(__uint_as_float(r.y << 16), a.z, acc); acc = fmaf(__uint_as_float(r.y & 0xffff0000u), a.w, acc);
    acc = fmaf(__uint_as_float(r.z << 16), b.x, acc); acc = fmaf(__uint_as_float(r.z & 0xffff0000u), b.y, acc);
    acc = fmaf(__uint_as_float(r.w << 16), b.z, acc); acc = fmaf(__uint_as_float(r.w & 0xffff0000u), b.w, acc);
    return acc;
  };
#pragma unroll
  for (int i = 0; i < PER; i++) {
    const int v = v0 + warp * PER + i;
    if (v >= sh.vdim) continue;  // warp-uniform
    const uint4 *w = reinterpret_cast<const uint4 *>(wuv + ((size_t)h * sh.vdim + v) * wuv_stride);
    float acc = 0.0f;
#pragma unroll
    for (int j = 0; j < PRE; j++)
      if (lane + 32 * j < pieces) acc = dot(pre[i][j], lane + 32 * j, acc);
    for (int k = lane + 32 * PRE; k < pieces; k += 32) acc = dot(__ldg(w + k), k, acc);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if (lane == 0) out[(size_t)h * sh.vdim + v] = acc * g;
  }
}

// ---- products of every head with its own matrix, f32: grid (column tiles, row tiles, heads) ----
constexpr int GP_M = 64, GP_N = 64, GP_K = 16;
__global__ void __launch_bounds__(256) grouped_product_kernel(const GroupedProduct p) {
  pdl_launch();
  pdl_wait();
  __shared__ float sx[GP_K][GP_M + 4], sw[GP_K][GP_N + 4];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4, z = blockIdx.z;
  const int m0 = blockIdx.y * GP_M, n0 = blockIdx.x * GP_N;
  const float *x = p.x + (size_t)z * p.x_z;
  const __nv_bfloat16 *w = p.w + (size_t)z * p.w_z;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += GP_K) {
    for (int i = tid; i < GP_M * GP_K; i += 256) {
      const int r = i / GP_K, k = i % GP_K;
      sx[k][r] = (m0 + r < p.rows && k0 + k < p.K) ? x[(size_t)(m0 + r) * p.x_row + k0 + k] : 0.0f;
      const int wr = p.w_k == 1 ? i / GP_K : i % GP_N, wk = p.w_k == 1 ? i % GP_K : i / GP_N;  // along the contiguous side
      sw[wk][wr] = (n0 + wr < p.N && k0 + wk < p.K) ? __bfloat162float(w[(size_t)(n0 + wr) * p.w_n + (size_t)(k0 + wk) * p.w_k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GP_K; k++) {
      float xv[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; i++) { xv[i] = sx[k][ty * 4 + i]; wv[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int r = m0 + ty * 4 + i;
    if (r >= p.rows) continue;
    const float g = p.gate ? lt_sigmoid(p.gate[(size_t)r * p.gate_stride + z]) : 1.0f;
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      const size_t off = (size_t)r * p.y_row + (size_t)z * p.y_z + n;
      if (p.y_bf16) reinterpret_cast<__nv_bfloat16 *>(p.y)[off] = __float2bfloat16_rn(acc[i][j] * g);
      else reinterpret_cast<float *>(p.y)[off] = acc[i][j] * g;
    }
  }
}

}  // namespace

dp_status dpk_latent_append(dp_ctx *ctx, const float *proj, int proj_stride, const LatentShape &sh, const __nv_bfloat16 *norm_w, const Rotation &rot,
                            const LatentCache &cache, float *q, float *q_rot, int rows, const RowMap &map) {
  if (cache.f32) DP_LAUNCH(ctx, latent_append_kernel<float>, rows, 256, 0, proj, proj_stride, sh, norm_w, rot, cache, q, q_rot, map);
  else DP_LAUNCH(ctx, latent_append_kernel<__half>, rows, 256, 0, proj, proj_stride, sh, norm_w, rot, cache, q, q_rot, map);
  return DP_OK;
}

dp_status dpk_latent_absorb_step(dp_ctx *ctx, const float *proj, const LatentShape &sh, const __nv_bfloat16 *norm_w, const Rotation &rot, const LatentCache &cache,
                                 const __nv_bfloat16 *wuk, int wuk_stride, const float *q, float *q_abs, const int *pos) {
  const dim3 grid(sh.heads + 1, (sh.kv_rank + LA_COLS - 1) / LA_COLS);
  if (cache.f32) DP_LAUNCH(ctx, latent_absorb_step_kernel<float>, grid, 256, 0, proj, sh, norm_w, rot, cache, wuk, wuk_stride, q, q_abs, pos);
  else DP_LAUNCH(ctx, latent_absorb_step_kernel<__half>, grid, 256, 0, proj, sh, norm_w, rot, cache, wuk, wuk_stride, q, q_abs, pos);
  return DP_OK;
}

dp_status dpk_latent_values_step(dp_ctx *ctx, const float *part, int splits, const LatentShape &sh, const __nv_bfloat16 *wuv, int wuv_stride, const float *gate,
                                 float *out) {
  const size_t smem = (size_t)wuv_stride * 4;
  if (smem > 48 * 1024) return dp_fail(ctx, DP_ERR_UNSUPPORTED, "latent attention: latent size %d", sh.kv_rank);
  DP_LAUNCH(ctx, latent_values_step_kernel, dim3(sh.heads, (sh.vdim + LV_ROWS - 1) / LV_ROWS), 256, smem, part, splits, sh, wuv, wuv_stride, gate, out);
  return DP_OK;
}

dp_status dpk_grouped_product(dp_ctx *ctx, const GroupedProduct &p) {
  DP_LAUNCH(ctx, grouped_product_kernel, dim3((p.N + GP_N - 1) / GP_N, (p.rows + GP_M - 1) / GP_M, p.heads), 256, 0, p);
  return DP_OK;
}
