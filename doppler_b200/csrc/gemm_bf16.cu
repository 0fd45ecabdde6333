// Products of several rows with bf16 weights: C [M, N] = A [M, K] W [N, K]^T, f32 accumulation and output.
//
// gemm_bf16_tc_kernel (bf16 activations): tcgen05 with both operands brought in by TMA.  The weights are the MMA's M
// side (128 output features), the activation rows its N side (16..256 of them, chosen at run time), so that few rows
// cost little and a row of TMEM lanes is a run of consecutive features: the epilogue stores 128 contiguous bytes per
// warp and activation row without staging.  Persistent: one CTA per SM walks the tiles; four roles (TMA, MMA issue,
// TMEM, four epilogue warps) with two accumulators in tensor memory, so the next tile's products run under this
// tile's stores.  K tails and rows beyond M or N are zero filled by TMA.  Every wait is bounded.
//
// gemm_bf16w_f32_kernel (f32 activations): the 32-bit mode.  bf16 weights are exact in f32; every product and sum is
// an f32 FMA on the CUDA cores.
//
// dpk_gemm_f16_tc: the same kernel with f16 operands and an f16 result.
//
// Optional decay: exp(-rate softplus(c + bias)) of every product is stored instead of the product.
// Optional gated activation: weight rows in groups of sixteen (eight gate rows, then their eight up rows) and
// g' sigmoid(slope g') (u' + shift) with g' = min(g, limit), u' = clamp(u, +-limit) stored in A's type.
#include "layers.h"
#include "pdl.cuh"
#include "umma.cuh"

#include <cstring>

using namespace umma;

namespace {

struct GluArgs {
  void *dst;
  int stride;
  float limit, slope, shift;
};

__device__ __forceinline__ float glu_act(float g, float u, const GluArgs &a) {
  if (a.limit > 0.0f) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit);
  }
  return g * (1.0f / (1.0f + expf(-a.slope * g))) * (u + a.shift);
}

// ... for a result that is stored as bf16
__device__ __forceinline__ float glu_act_fast(float g, float u, const GluArgs &a) {
  if (a.limit > 0.0f) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit);
  }
  return __fdividef(g, 1.0f + __expf(-a.slope * g)) * (u + a.shift);
}

__device__ __forceinline__ float decay_of(float c, float rate, float bias) {
  const float z = c + bias;
  return expf(-rate * (fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)))));
}

constexpr int BT_THREADS = 256, BT_MAX_STAGES = 8;
constexpr uint32_t BT_W_TILE = 128u * 128u;  // 128 weight rows x 64 bf16

struct TcArgs {
  float *C;
  __half *C16;   // f16 operands and result (rows of c_stride elements)
  int M, N, K, bn, stages, tiles_n, tiles_m, tmem_cols, c_stride;
  GluArgs glu;
  DecayOut decay;
};

__device__ __forceinline__ uint32_t idesc_16(int M, int N, bool f16) {  // D = f32, A = B = bf16 or f16, both K-major
  return (1u << 4) | (f16 ? 0u : (1u << 7) | (1u << 10)) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(M >> 4) << 24);
}

__global__ void __launch_bounds__(BT_THREADS, 1) gemm_bf16_tc_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_a,
                                                                     const TcArgs a, int *__restrict__ err) {
  extern __shared__ uint8_t bt_raw[];
  uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(bt_raw) + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) uint64_t bars[2 * BT_MAX_STAGES + 4];
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_word;
  volatile int *abort_flag = &abort_word;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int S = a.stages;
  const uint32_t stage_bytes = BT_W_TILE + (uint32_t)a.bn * 128u;
  const uint32_t bar0 = smem_u32(bars);
  auto full = [&](int s) { return bar0 + 8u * (uint32_t)s; };
  auto empty = [&](int s) { return bar0 + 8u * (uint32_t)(BT_MAX_STAGES + s); };
  auto acc_full = [&](int b) { return bar0 + 8u * (uint32_t)(2 * BT_MAX_STAGES + b); };
  auto acc_empty = [&](int b) { return bar0 + 8u * (uint32_t)(2 * BT_MAX_STAGES + 2 + b); };
  const int tiles = a.tiles_n * a.tiles_m, ksteps = (a.K + BK - 1) / BK;

  pdl_launch();
  pdl_wait();
  if (tid == 0) {
    for (int s = 0; s < S; s++) { mbar_init(full(s), 1); mbar_init(empty(s), 1); }
    for (int b = 0; b < 2; b++) { mbar_init(acc_full(b), 1); mbar_init(acc_empty(b), 4); }
    abort_word = 0;
    mbar_fence_init();
  }
  if (warp == 2) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"((uint32_t)a.tmem_cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t *>(&tmem_slot);

  if (warp == 0) {
    if (lane == 0) {
      uint32_t it = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x) {
        const int n0 = (tile / a.tiles_m) * 128, m0 = (tile % a.tiles_m) * a.bn;
        for (int k = 0; k < ksteps; k++, it++) {
          const int s = (int)(it % (uint32_t)S);
          if (it >= (uint32_t)S && !mbar_wait_bounded(empty(s), ((it / (uint32_t)S) - 1u) & 1u, abort_flag)) { ok = false; break; }
          mbar_expect_tx(full(s), stage_bytes);
          const uint32_t dst = smem_u32(smem) + (uint32_t)s * stage_bytes;
          tma_load_2d(dst, &tmap_w, k * BK, n0, full(s));
          tma_load_2d(dst + BT_W_TILE, &tmap_a, k * BK, m0, full(s));
        }
      }
      // no copy may still be in flight when the CTA ends, also where a wait gave up
      const uint32_t held = it < (uint32_t)S ? it : (uint32_t)S;
      for (uint32_t i = it - held; i < it; i++)
        for (uint32_t poll = 0; poll < (1u << 20) && !mbar_try_wait(full((int)(i % (uint32_t)S)), (i / (uint32_t)S) & 1u); poll++) {}
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = idesc_16(128, a.bn, a.C16 != nullptr);
      uint32_t it = 0, n = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, n++) {
        const int b = (int)(n & 1u);
        if (n >= 2 && !mbar_wait_bounded(acc_empty(b), ((n >> 1) - 1u) & 1u, abort_flag)) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t acc = tmem + (uint32_t)(b * a.bn);
        for (int k = 0; k < ksteps; k++, it++) {
          const int s = (int)(it % (uint32_t)S);
          if (!mbar_wait_bounded(full(s), (it / (uint32_t)S) & 1u, abort_flag)) { ok = false; break; }
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          const uint32_t w_addr = smem_u32(smem) + (uint32_t)s * stage_bytes, x_addr = w_addr + BT_W_TILE;
#pragma unroll
          for (int k16 = 0; k16 < BK / 16; k16++)
            umma_f16(acc, umma_desc_sw128(w_addr + (uint32_t)k16 * 32u), umma_desc_sw128(x_addr + (uint32_t)k16 * 32u), idesc, (k > 0 || k16 > 0) ? 1u : 0u);
          umma_commit(empty(s));
        }
        if (ok) umma_commit(acc_full(b));
      }
    }
  } else if (warp >= 4) {
    const int quad = warp & 3;
    uint32_t n = 0;
    for (int tile = blockIdx.x; tile < tiles; tile += gridDim.x, n++) {
      const int b = (int)(n & 1u);
      const int n0 = (tile / a.tiles_m) * 128, m0 = (tile % a.tiles_m) * a.bn;
      const bool ready = mbar_wait_bounded(acc_full(b), (n >> 1) & 1u, abort_flag);
      if (!__all_sync(0xffffffffu, ready)) break;  // tcgen05.ld is warp-wide: together or not at all
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const int f = n0 + quad * 32 + lane;
      const uint32_t taddr = tmem + ((uint32_t)(quad * 32) << 16) + (uint32_t)(b * a.bn);
      for (int c0 = 0; c0 < a.bn; c0 += 16) {
        if (m0 + c0 >= a.M) break;  // (uniform) no such activation rows
        uint32_t r[16];
        tmem_ld16(taddr + (uint32_t)c0, r);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        if (a.glu.dst) {
          // a gate row and its up row are eight lanes apart: the gate's lane takes the even activation rows of the pair,
          // the other lane the odd ones
          const bool is_up = lane & 8;
          __nv_bfloat16 *dst = reinterpret_cast<__nv_bfloat16 *>(a.glu.dst) + (f >> 4) * 8 + (f & 7);
#pragma unroll
          for (int i = 0; i < 16; i += 2) {
            const float got = __shfl_xor_sync(0xffffffffu, __uint_as_float(is_up ? r[i] : r[i + 1]), 8);
            const float gv = is_up ? got : __uint_as_float(r[i]), uv = is_up ? __uint_as_float(r[i + 1]) : got;
            const int row = m0 + c0 + i + (is_up ? 1 : 0);
            if (f < a.N && row < a.M) dst[(size_t)row * a.glu.stride] = __float2bfloat16_rn(glu_act_fast(gv, uv, a.glu));
          }
        } else if (a.C16) {
          if (f < a.N) {
            __half *dst = a.C16 + (size_t)(m0 + c0) * a.c_stride + f;
#pragma unroll
            for (int i = 0; i < 16; i++)
              if (m0 + c0 + i < a.M) dst[(size_t)i * a.c_stride] = __float2half_rn(__uint_as_float(r[i]));
          }
        } else if (f < a.N) {
          if (a.decay.rate) {
            const float rate = a.decay.rate[f], bias = a.decay.bias[f];
#pragma unroll 4
            for (int i = 0; i < 16; i++) r[i] = __float_as_uint(decay_of(__uint_as_float(r[i]), rate, bias));
          }
          float *dst = a.C + (size_t)(m0 + c0) * a.N + f;
#pragma unroll
          for (int i = 0; i < 16; i++)
            if (m0 + c0 + i < a.M) dst[(size_t)i * a.N] = __uint_as_float(r[i]);
        }
      }
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(acc_empty(b));
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 2) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((uint32_t)a.tmem_cols) : "memory");
  if (abort_word && tid == 0) atomicExch(err, 2);
}

// ---- 32-bit mode ----
constexpr int FM = 64, FN = 64, FK = 16;
__global__ void __launch_bounds__(256) gemm_bf16w_f32_kernel(const __nv_bfloat16 *__restrict__ W, int w_stride, const float *__restrict__ A, int a_stride,
                                                             float *__restrict__ C, int M, int N, int K, const GluArgs glu, const DecayOut decay) {
  pdl_launch();
  pdl_wait();
  __shared__ float sa[FK][FM + 4], sw[FK][FN + 4];
  __shared__ float sc[FM][FN + 1];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int m0 = blockIdx.y * FM, n0 = blockIdx.x * FN;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += FK) {
    for (int i = tid; i < FM * FK; i += 256) {
      const int r = i / FK, k = i % FK;
      sa[k][r] = (m0 + r < M && k0 + k < K) ? A[(size_t)(m0 + r) * a_stride + k0 + k] : 0.0f;
      sw[k][r] = (n0 + r < N && k0 + k < K) ? __bfloat162float(W[(size_t)(n0 + r) * w_stride + k0 + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < FK; k++) {
      float av[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; i++) { av[i] = sa[k][ty * 4 + i]; wv[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
  if (!glu.dst) {
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
      for (int j = 0; j < 4; j++)
        if (m0 + ty * 4 + i < M && n0 + tx * 4 + j < N) {
          const int n = n0 + tx * 4 + j;
          C[(size_t)(m0 + ty * 4 + i) * N + n] = decay.rate ? decay_of(acc[i][j], decay.rate[n], decay.bias[n]) : acc[i][j];
        }
    return;
  }
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) sc[ty * 4 + i][tx * 4 + j] = acc[i][j];
  __syncthreads();
  for (int i = tid; i < FM * FN / 2; i += 256) {
    const int r = i / (FN / 2), o = i % (FN / 2), c = (o >> 3) * 16 + (o & 7);
    if (m0 + r < M && n0 + c < N)
      reinterpret_cast<float *>(glu.dst)[(size_t)(m0 + r) * glu.stride + n0 / 2 + o] = glu_act(sc[r][c], sc[r][c + 8], glu);
  }
}

GluArgs glu_args(const GluOut *g) {
  GluArgs a = {nullptr, 0, 0.0f, 0.0f, 0.0f};
  if (g) { a.dst = g->dst; a.stride = g->stride; a.limit = g->limit; a.slope = g->slope; a.shift = g->shift; }
  return a;
}

// activation rows per tile: the width with the least (waves x (products of a tile + its fixed cost))
int pick_rows(dp_ctx *ctx, int M, int tiles_n) {
  int best = 16;
  double best_cost = -1.0;
  for (int bn = 16; bn <= 256; bn += 16) {
    const long tiles = (long)tiles_n * ((M + bn - 1) / bn);
    const long waves = (tiles + ctx->sm_count - 1) / ctx->sm_count;
    // tiles narrower than 128 rows are paced by the weight operand's shared-memory reads, not by the products
    const double cost = (double)waves * ((bn < 128 ? 128 : bn) + 16);
    if (best_cost < 0 || cost < best_cost) { best = bn; best_cost = cost; }
  }
  return best;
}

// shape, strides and outputs are in `a`; the rest is chosen here
dp_status launch_tc(dp_ctx *ctx, const void *W, int w_stride, const void *A, int a_stride, TcArgs a) {
  const int M = a.M, N = a.N, K = a.K;
  DP_CHECK(ctx, w_stride % 8 == 0 && a_stride % 8 == 0 && K <= w_stride && K <= a_stride && M > 0 && N > 0 && K > 0, "gemm (bf16): bad shape or stride");
  EncodeTiledFn encode = get_encode();
  if (!encode) return dp_fail(ctx, DP_ERR_CUDA, "gemm (bf16): cuTensorMapEncodeTiled is not available");
  a.tiles_n = (N + 127) / 128;
  a.bn = pick_rows(ctx, M, a.tiles_n);
  a.tiles_m = (M + a.bn - 1) / a.bn;
  const uint32_t stage_bytes = BT_W_TILE + (uint32_t)a.bn * 128u;
  const size_t budget = ctx->smem_optin - 2048;
  int stages = (int)((budget - 1024) / stage_bytes);
  if (stages > BT_MAX_STAGES) stages = BT_MAX_STAGES;
  a.stages = stages;
  a.tmem_cols = 32;
  while (a.tmem_cols < 2 * a.bn) a.tmem_cols *= 2;
  const CUtensorMapDataType type = a.C16 ? CU_TENSOR_MAP_DATA_TYPE_FLOAT16 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  CUtensorMap tw, ta;
  const cuuint32_t estr[2] = {1, 1};
  const cuuint64_t wd[2] = {(cuuint64_t)K, (cuuint64_t)N}, ad[2] = {(cuuint64_t)K, (cuuint64_t)M};
  const cuuint64_t ws[1] = {(cuuint64_t)w_stride * 2}, as[1] = {(cuuint64_t)a_stride * 2};
  const cuuint32_t wb[2] = {BK, 128}, ab[2] = {BK, (cuuint32_t)a.bn};
  CUresult r = encode(&tw, type, 2, (void *)W, wd, ws, wb, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                      CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r == CUDA_SUCCESS)
    r = encode(&ta, type, 2, (void *)A, ad, as, ab, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
               CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return dp_fail(ctx, DP_ERR_CUDA, "gemm (bf16): cuTensorMapEncodeTiled failed (%d) for [%d,%d] x [%d,%d]", (int)r, M, K, N, K);
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    DP_CUDA(ctx, cudaFuncSetAttribute(gemm_bf16_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)budget));
    attr.done(ctx->device);
  }
  const int tiles = a.tiles_n * a.tiles_m, grid = tiles < ctx->sm_count ? tiles : ctx->sm_count;
  DP_LAUNCH(ctx, gemm_bf16_tc_kernel, grid, BT_THREADS, (size_t)stages * stage_bytes + 1024, tw, ta, a, ctx->dev_status);
  return DP_OK;
}

}  // namespace

dp_status dpk_gemm_bf16_tc(dp_ctx *ctx, const __nv_bfloat16 *W, int w_stride, const __nv_bfloat16 *A, int a_stride, float *C, int M, int N, int K,
                           const GluOut *glu, const DecayOut *decay) {
  DP_CHECK(ctx, !glu || N % 16 == 0, "gemm (bf16): gate and up rows come in groups of sixteen");
  TcArgs a = {};
  a.C = C; a.M = M; a.N = N; a.K = K;
  a.glu = glu_args(glu);
  if (decay) a.decay = *decay;
  return launch_tc(ctx, W, w_stride, A, a_stride, a);
}

dp_status dpk_gemm_f16_tc(dp_ctx *ctx, const __half *W, int w_stride, const __half *A, int a_stride, __half *C, int c_stride, int M, int N, int K) {
  TcArgs a = {};
  a.C16 = C; a.c_stride = c_stride; a.M = M; a.N = N; a.K = K;
  return launch_tc(ctx, W, w_stride, A, a_stride, a);
}

dp_status dpk_gemm_bf16w_f32(dp_ctx *ctx, const __nv_bfloat16 *W, int w_stride, const float *A, int a_stride, float *C, int M, int N, int K,
                             const GluOut *glu, const DecayOut *decay) {
  DP_CHECK(ctx, M > 0 && N > 0 && K > 0, "gemm (bf16 weights, f32): bad shape");
  DP_CHECK(ctx, !glu || N % 16 == 0, "gemm (bf16): gate and up rows come in groups of sixteen");
  DP_LAUNCH(ctx, gemm_bf16w_f32_kernel, dim3((N + FN - 1) / FN, (M + FM - 1) / FM), 256, 0, W, w_stride, A, a_stride, C, M, N, K, glu_args(glu),
            decay ? *decay : DecayOut());
  return DP_OK;
}
