// Attention on a latent cache (f16 rows that all query heads share; the values are the first part of the keys) for single
// query rows: decode steps and short portions, split over the keys like attention_tc.cu, partials (o, m, l) per split.
//
//   S = Q K^T   M = 16 query heads, N = keys, K = the row (latent | rotated part)
//   O = P C     M = 16 query heads, N = latent values, K = keys
//
// A row is long (hundreds of values) and used by every head, so the warps of a CTA split the work differently in the two
// products: for S a warp owns every eighth step of sixteen row values, its share of Q stays in registers (f16 hi and lo
// halves, S in f32 accumulators) and the eight partial tiles are added through shared memory; for O a warp owns every
// eighth run of sixteen latent values.  Either way a cached value is read from shared memory by one warp only.  P enters as
// f16 hi and lo halves too.  64 keys at a time, two stages filled with cp.async.
#include "attn_out.cuh"
#include "common.h"
#include "pdl.cuh"

#include <cfloat>
#include <cmath>

namespace {

constexpr int AL_WARPS = 8, AL_THREADS = AL_WARPS * 32, AL_KEYS = 64, AL_HEADS = 16;
constexpr int AL_SPITCH = AL_KEYS + 4;      // floats per row of a partial score tile
constexpr int AL_PPITCH = AL_KEYS * 2 + 16; // bytes per row of P

__device__ __forceinline__ uint32_t al_smem(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void al_ldm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void al_ldmt(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void al_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two f32 values as packed f16 pairs hi + lo
__device__ __forceinline__ void al_split(float x, float y, uint32_t &hi, uint32_t &lo) {
  const __half2 h = __floats2half2_rn(x, y);
  const float2 f = __half22float2(h);
  const __half2 l = __floats2half2_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t *>(&h);
  lo = *reinterpret_cast<const uint32_t *>(&l);
}

// KS: steps of sixteen row values per warp, NU: runs of sixteen latent values per warp
template <int KS, int NU>
__global__ void __launch_bounds__(AL_THREADS, 1) attn_latent_kernel(const dpk_attn_params p, float *__restrict__ part, int splits) {
  pdl_launch();
  pdl_wait();
  extern __shared__ __align__(128) unsigned char al_raw[];
  __shared__ float s_alpha[AL_HEADS], s_m[AL_HEADS], s_l[AL_HEADS];
  const int D = p.head_dim, V = p.v_dim, row_b = D * 2 + 16, pieces = D / 8, k_steps = D / 16, v_units = V / 16;
  const int stage_b = AL_KEYS * row_b;
  float *s_part = reinterpret_cast<float *>(al_raw + 2 * stage_b);  // [warp][16][AL_SPITCH]
  unsigned char *s_p = reinterpret_cast<unsigned char *>(s_part + AL_WARPS * AL_HEADS * AL_SPITCH);  // P hi, P lo [16][AL_PPITCH]
  const uint32_t sm = al_smem(al_raw), sm_p = al_smem(s_p);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int split = blockIdx.x, h0 = blockIdx.y * AL_HEADS, z = blockIdx.z, b = z / p.seq_len, qi = z % p.seq_len;
  const int kv_len = p.kv_lens ? min(max(p.kv_lens[b], 0), p.kv_len) : p.kv_len;
  const AttnRange range = attn_range(p, kv_len, qi);
  const int per_split = (range.hi - range.lo + splits - 1) / splits;
  const int k_begin = range.lo + split * per_split, k_end = min(k_begin + per_split, range.hi);
  const int tiles = k_end > k_begin ? (k_end - k_begin + AL_KEYS - 1) / AL_KEYS : 0;
  const __half *rows = p.k + (size_t)b * p.kv_batch_stride;

  auto stage = [&](int tile) {
    if (tile < tiles) {
      const uint32_t dst = sm + (uint32_t)(tile & 1) * stage_b;
      const int key0 = k_begin + tile * AL_KEYS;
      for (int r = warp; r < AL_KEYS; r += AL_WARPS) {
        const bool ok = key0 + r < k_end;
        const __half *src = rows + (size_t)(ok ? key0 + r : k_begin) * p.v_row_stride;
        for (int c = lane; c < pieces; c += 32)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + r * row_b + c * 16), "l"(src + c * 8), "r"(ok ? 16 : 0) : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  stage(0);

  // this warp's share of Q, times scale log2(e)
  const float qmul = p.scale * 1.4426950408889634f;
  uint32_t qh[KS][4], ql[KS][4];
#pragma unroll
  for (int i = 0; i < KS; i++) {
    const int ks = warp + AL_WARPS * i;
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int head = h0 + g + (j & 1) * 8, d = ks * 16 + 2 * t4 + (j >> 1) * 8;
      float2 x = make_float2(0.0f, 0.0f);
      if (ks < k_steps && head < p.num_heads) x = *reinterpret_cast<const float2 *>(p.q + ((size_t)z * p.num_heads + head) * D + d);
      al_split(x.x * qmul, x.y * qmul, qh[i][j], ql[i][j]);
    }
  }
  float o[NU][2][4];
#pragma unroll
  for (int i = 0; i < NU; i++)
#pragma unroll
    for (int j = 0; j < 2; j++) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.0f;
  const int my_row = tid >> 4, my_key = (tid & 15) * 4;  // softmax: sixteen threads per head, four keys each
  float m_run = -INFINITY, l_run = 0.0f;

  for (int tile = 0; tile < tiles; tile++) {
    stage(tile + 1);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const uint32_t base = sm + (uint32_t)(tile & 1) * stage_b;
    // ---- S, this warp's steps ----
    float s[8][4];
#pragma unroll
    for (int n = 0; n < 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.0f;
#pragma unroll
    for (int i = 0; i < KS; i++) {
      const int ks = warp + AL_WARPS * i;
      if (ks < k_steps) {
#pragma unroll
        for (int n = 0; n < 4; n++) {  // sixteen keys
          uint32_t r[4];
          al_ldm(r, base + (n * 16 + (lane & 7) + 8 * (lane >> 4)) * row_b + ks * 32 + ((lane >> 3) & 1) * 16);
          al_mma(s[2 * n], qh[i], r[0], r[1]);
          al_mma(s[2 * n + 1], qh[i], r[2], r[3]);
          al_mma(s[2 * n], ql[i], r[0], r[1]);
          al_mma(s[2 * n + 1], ql[i], r[2], r[3]);
        }
      }
    }
    float *sp = s_part + warp * AL_HEADS * AL_SPITCH;
#pragma unroll
    for (int n = 0; n < 8; n++) {
      *reinterpret_cast<float2 *>(sp + g * AL_SPITCH + n * 8 + 2 * t4) = make_float2(s[n][0], s[n][1]);
      *reinterpret_cast<float2 *>(sp + (g + 8) * AL_SPITCH + n * 8 + 2 * t4) = make_float2(s[n][2], s[n][3]);
    }
    __syncthreads();
    // ---- softmax ----
    {
      float x[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
      for (int w = 0; w < AL_WARPS; w++) {
        const float4 v = *reinterpret_cast<const float4 *>(s_part + (w * AL_HEADS + my_row) * AL_SPITCH + my_key);
        x[0] += v.x; x[1] += v.y; x[2] += v.z; x[3] += v.w;
      }
      const int key0 = k_begin + tile * AL_KEYS + my_key;
      float mx = -INFINITY;
#pragma unroll
      for (int j = 0; j < 4; j++) {
        if (key0 + j >= k_end) x[j] = -INFINITY;
        mx = fmaxf(mx, x[j]);
      }
#pragma unroll
      for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_new = fmaxf(m_run, mx);  // finite: a tile holds a key
      const float alpha = exp2f(m_run - m_new);
      m_run = m_new;
      float e[4], sum = 0.0f;
#pragma unroll
      for (int j = 0; j < 4; j++) { e[j] = exp2f(x[j] - m_new); sum += e[j]; }
      l_run = l_run * alpha + sum;
      if ((tid & 15) == 0) s_alpha[my_row] = alpha;
      uint32_t hi[2], lo[2];
      al_split(e[0], e[1], hi[0], lo[0]);
      al_split(e[2], e[3], hi[1], lo[1]);
      *reinterpret_cast<uint2 *>(s_p + my_row * AL_PPITCH + my_key * 2) = make_uint2(hi[0], hi[1]);
      *reinterpret_cast<uint2 *>(s_p + (AL_HEADS + my_row) * AL_PPITCH + my_key * 2) = make_uint2(lo[0], lo[1]);
    }
    __syncthreads();
    // ---- O, this warp's runs ----
    const float al0 = s_alpha[g], al1 = s_alpha[g + 8];
#pragma unroll
    for (int i = 0; i < NU; i++)
#pragma unroll
      for (int j = 0; j < 2; j++) { o[i][j][0] *= al0; o[i][j][1] *= al0; o[i][j][2] *= al1; o[i][j][3] *= al1; }
#pragma unroll
    for (int k = 0; k < AL_KEYS / 16; k++) {
      uint32_t ph[4], pl[4];
      const uint32_t pa = sm_p + (lane & 15) * AL_PPITCH + k * 32 + (lane >> 4) * 16;
      al_ldm(ph, pa);
      al_ldm(pl, pa + AL_HEADS * AL_PPITCH);
#pragma unroll
      for (int i = 0; i < NU; i++) {
        const int u = warp + AL_WARPS * i;
        if (u < v_units) {
          uint32_t r[4];
          al_ldmt(r, base + (k * 16 + (lane & 15)) * row_b + u * 32 + (lane >> 4) * 16);
          al_mma(o[i][0], ph, r[0], r[1]);
          al_mma(o[i][1], ph, r[2], r[3]);
          al_mma(o[i][0], pl, r[0], r[1]);
          al_mma(o[i][1], pl, r[2], r[3]);
        }
      }
    }
    __syncthreads();  // the stage is refilled after the next round's start, P and the partial scores are rewritten
  }
#pragma unroll
  for (int off = 8; off > 0; off >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, off);
  if ((tid & 15) == 0) { s_m[my_row] = m_run == -INFINITY ? -FLT_MAX : m_run; s_l[my_row] = l_run; }
  __syncthreads();
#pragma unroll
  for (int half = 0; half < 2; half++) {
    const int head = h0 + g + 8 * half;
    if (head >= p.num_heads) continue;
    const float l = s_l[g + 8 * half], inv = splits > 1 ? 1.0f : (l > 0.0f ? 1.0f / l : 0.0f);
    float *dst = splits > 1 ? part + (((size_t)z * p.num_heads + head) * splits + split) * (V + 2) : p.out + ((size_t)z * p.num_heads + head) * V;
#pragma unroll
    for (int i = 0; i < NU; i++) {
      const int u = warp + AL_WARPS * i;
      if (u >= v_units) continue;
#pragma unroll
      for (int j = 0; j < 2; j++)
        *reinterpret_cast<float2 *>(dst + u * 16 + j * 8 + 2 * t4) = make_float2(o[i][j][2 * half] * inv, o[i][j][2 * half + 1] * inv);
    }
    if (splits > 1 && warp == 0 && t4 == 0) { dst[V] = s_m[g + 8 * half]; dst[V + 1] = l; }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
}

size_t latent_smem(const dpk_attn_params &p) {
  return (size_t)2 * AL_KEYS * (p.head_dim * 2 + 16) + (size_t)AL_WARPS * AL_HEADS * AL_SPITCH * 4 + 2 * AL_HEADS * AL_PPITCH;
}

template <int KS, int NU>
dp_status launch(dp_ctx *ctx, const dpk_attn_params &p, float *scratch, int splits) {
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    DP_CUDA(ctx, cudaFuncSetAttribute((attn_latent_kernel<KS, NU>), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ctx->smem_optin - 1024));
    attr.done(ctx->device);
  }
  const dim3 grid(splits, (p.num_heads + AL_HEADS - 1) / AL_HEADS, p.batch * p.seq_len);
  DP_LAUNCH(ctx, (attn_latent_kernel<KS, NU>), grid, AL_THREADS, latent_smem(p), p, scratch, splits);
  return DP_OK;
}

}  // namespace

// f16 rows shared by all heads, values their first v_dim elements, both sizes multiples of sixteen
bool dpk_attention_latent_eligible(dp_ctx *ctx, const dpk_attn_params &p) {
  if (p.kv_f32 || p.num_kv_heads != 1 || p.v_row_stride != p.head_dim || p.v != p.k || p.v_dim <= 0) return false;
  if (p.head_dim % 16 || p.v_dim % 16 || p.v_dim > p.head_dim || p.head_dim > 5 * 128 || p.v_dim > 4 * 128) return false;
  if (p.softcap > 0.0f || p.gate || p.out_bf16 || p.fuse.qkv || p.chunk || p.sliding_window) return false;
  if (p.kv_batch_stride % 8 || ((uintptr_t)p.k & 15) || ((uintptr_t)p.q & 7) || ((uintptr_t)p.out & 7)) return false;
  return latent_smem(p) + 1024 <= ctx->smem_optin;
}

// splits: the CTAs of one wave, at least one tile of keys each
int dpk_attention_latent_splits(dp_ctx *ctx, const dpk_attn_params &p) {
  const long base = (long)p.batch * p.seq_len * ((p.num_heads + AL_HEADS - 1) / AL_HEADS);
  long s = ctx->sm_count / base, most = (p.kv_len + AL_KEYS - 1) / AL_KEYS;
  if (s > most) s = most;
  if (s > 32) s = 32;
  return s < 1 ? 1 : (int)s;
}

dp_status dpk_attention_latent(dp_ctx *ctx, const dpk_attn_params &p, float *scratch, int splits) {
  if (p.head_dim <= 256 && p.v_dim <= 256) return launch<2, 2>(ctx, p, scratch, splits);
  return launch<5, 4>(ctx, p, scratch, splits);
}
