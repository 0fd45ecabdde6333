// Mamba-2 recurrence over a portion of a prompt in chunks of 64 tokens, on the tensor cores.
//
// With c_t the running sum of a dt within the chunk (a = -exp(A_log), or ln(decay) with dt = 1) and S the state before it, the recurrence unrolls to
//   y_t = exp(c_t) S^T C_t + sum_{s <= t} exp(c_t - c_s) dt_s (C_t . B_s) x_s
//   S'  = exp(c_end) S + sum_s exp(c_end - c_s) dt_s B_s x_s^T
// (the chunked form of Dao and Gu, "Transformers are SSMs", 2024).  x, B and C, the activations of the short
// convolution, are bf16; everything else is f32: sums are f32 accumulators, the state lives in f32 registers, and an
// f32 operand (the state, the weighted C.B products, the weighted x) enters its product as three bf16 terms that add
// up to its 24 bits, each multiplied exactly with the bf16 operand.
//
// One CTA = PB of a head's value columns, chunks in sequence.  Per chunk, with mma.sync m16n8k16:
//   Xw [s, p] = exp(c_end - c_s) dt_s x_s  split, to shared memory
//   G  [t, s] = C B^T                 each warp a block of it; weighted, split, to shared memory
//   Y^T[p, t] = S^T C^T (state terms from shared memory), scaled by exp(c_t), then += X^T G'^T
//   S^T[p, n] = exp(c_end) S^T + Xw^T B   in registers; its terms go to shared memory for the next chunk
// with the warps dealt (16 p) x (64 / TW t) for Y and (16 p) x (N / TW n) for S.  The next chunk's rows are brought in
// with cp.async meanwhile.  Shared rows are padded by 16 bytes, which makes every ldmatrix conflict free.
#include "layers.h"
#include "pdl.cuh"

namespace {

constexpr int CQ = 64, TERMS = 3;

__device__ __forceinline__ uint32_t ck_smem(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ck_cp16(uint32_t dst, const void *src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void ck_ldm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ck_ldm2(uint32_t &r0, uint32_t &r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ck_ldmt(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ck_ldmt2(uint32_t &r0, uint32_t &r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ck_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// B fragments (one k step of 16) of T tiles of eight rows, rows of `pitch` bytes from addr on
template <int T> __device__ __forceinline__ void ck_load_b(uint32_t (&b)[T][2], uint32_t addr, int pitch, int lane) {
  if constexpr (T % 2 == 0) {
#pragma unroll
    for (int j = 0; j < T / 2; j++) {
      uint32_t r[4];
      ck_ldm(r, addr + (j * 16 + (lane & 7) + 8 * (lane >> 4)) * pitch + ((lane >> 3) & 1) * 16);
      b[2 * j][0] = r[0]; b[2 * j][1] = r[1]; b[2 * j + 1][0] = r[2]; b[2 * j + 1][1] = r[3];
    }
  } else {
    ck_ldm2(b[0][0], b[0][1], addr + (lane & 7) * pitch + ((lane >> 3) & 1) * 16);
  }
}
// two f32 values as TERMS packed bf16 pairs whose sums are the values
__device__ __forceinline__ void ck_split(float x, float y, uint32_t (&t)[TERMS]) {
#pragma unroll
  for (int i = 0; i < TERMS; i++) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    t[i] = *reinterpret_cast<const uint32_t *>(&h);
    x -= __uint_as_float(t[i] << 16);
    y -= __uint_as_float(t[i] & 0xffff0000u);
  }
}
__device__ __forceinline__ float ck_exp2(float v) {  // relative error 2^-22
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}
__device__ __forceinline__ float ck_silu(float v) { return __fdividef(v, 1.0f + __expf(-v)); }  // the output gate, not the recurrence

template <int N, int PB> struct CkLayout {
  static constexpr int NROW = N * 2 + 16, QROW = CQ * 2 + 16, PROW = PB * 2 + 16;  // bytes per shared row
  static constexpr int B = 0, C = B + CQ * NROW, X = C + CQ * NROW, DT = X + CQ * PROW, STAGE = DT + CQ * 4;
  static constexpr int WARPS = PB > 32 ? 16 : 8, THREADS = WARPS * 32;
  static constexpr int STAGES = PB > 32 ? 2 : 1;      // one, where that lets two CTAs share an SM
  static constexpr int M = STAGES * STAGE;                 // weighted C.B terms [TERMS][t][s]
  static constexpr int S = M + TERMS * CQ * QROW;     // state terms [TERMS][p][n]
  static constexpr int XW = S + TERMS * PB * NROW;    // weighted x terms [TERMS][s][p]
  static constexpr int CUM = XW + TERMS * CQ * PROW;   // c_t log2(e), then the weights of the state update
  static constexpr int TOTAL = CUM + 2 * CQ * 4;
};

template <int N, int PB>
__global__ void __launch_bounds__((CkLayout<N, PB>::THREADS), PB > 32 ? 1 : 2) ssm_chunk_kernel(const float *__restrict__ proj, int proj_stride, const __nv_bfloat16 *__restrict__ xbc,
                                                               const float *__restrict__ dt, const SsmShape sh, const SsmWeights w, const SsmState st,
                                                               float *__restrict__ out, int rows, int start_pos, int seq) {
  pdl_launch();
  pdl_wait();
  using L = CkLayout<N, PB>;
  constexpr int PBLK = PB / 16, TW = L::WARPS / PBLK;  // p blocks, warps per p block
  constexpr int TT = CQ / TW / 8;                      // 8-token tiles of Y per warp
  constexpr int NTILES = N / 8, NT = NTILES >= TW ? NTILES / TW : 1;  // 8-wide state tiles per warp
  extern __shared__ __align__(128) unsigned char ck_raw[];
  const uint32_t sm = ck_smem(ck_raw);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.x, p0 = blockIdx.y * PB;
  const int P = sh.vdim, G = sh.groups, inner = sh.heads * P, CH = inner + 2 * G * N;
  const int grp = h / (sh.heads / G);
  const int pblk = warp / TW, tw = warp % TW;
  const int chunks = (rows + CQ - 1) / CQ;
  const float a2 = w.a[h] * 1.4426950408889634f, dh = w.d ? w.d[h] : 0.0f;
  float *s_cum = reinterpret_cast<float *>(ck_raw + L::CUM), *s_wt = s_cum + CQ;

  auto stage = [&](int chunk) {
    const uint32_t base = sm + (uint32_t)(chunk % L::STAGES) * L::STAGE;
    const int r0 = chunk * CQ;
    constexpr int CB = N / 8, CX = PB / 8;  // 16-byte pieces per token
    // B and C: a warp per token, a lane per piece
    if (lane < 2 * CB) {
      const bool is_c = lane >= CB;
      const int e = is_c ? lane - CB : lane;
      const __nv_bfloat16 *src = xbc + inner + ((is_c ? G : 0) + grp) * N + e * 8;
      const uint32_t dst = base + (is_c ? L::C : L::B) + e * 16;
#pragma unroll
      for (int t = warp; t < CQ; t += L::WARPS) {
        const bool ok = r0 + t < rows;
        ck_cp16(dst + t * L::NROW, src + (size_t)(ok ? r0 + t : 0) * CH, ok ? 16 : 0);
      }
    }
    if (tid < CQ * CX) {
      const int t = tid / CX, e = tid % CX;
      const bool ok = r0 + t < rows;
      ck_cp16(base + L::X + t * L::PROW + e * 16, xbc + (size_t)(ok ? r0 + t : 0) * CH + h * P + p0 + e * 8, ok ? 16 : 0);
    }
    if (tid < CQ) {
      const bool ok = r0 + tid < rows;
      if (w.decay) *reinterpret_cast<float *>(ck_raw + (base - sm) + L::DT + tid * 4) = ok ? 1.0f : 0.0f;
      else asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(base + L::DT + tid * 4), "l"(dt + (size_t)(ok ? r0 + tid : 0) * sh.heads + h),
                   "r"(ok ? 4 : 0) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // state accumulators: rows p (g, g + 8) of this warp's p block, columns n of its slice
  float acc_s[NT][4];
  const bool has_state = tw * NT < NTILES;
  float *S0 = st.s + (size_t)seq * st.s_seq + ((size_t)h * P + p0 + pblk * 16 + g) * N + (has_state ? tw * NT * 8 : 0) + 2 * t4;
#pragma unroll
  for (int j = 0; j < NT; j++) {
    float2 v0 = make_float2(0.0f, 0.0f), v1 = v0;
    if (start_pos > 0 && has_state) {
      v0 = *reinterpret_cast<const float2 *>(S0 + j * 8);
      v1 = *reinterpret_cast<const float2 *>(S0 + 8 * N + j * 8);
    }
    acc_s[j][0] = v0.x; acc_s[j][1] = v0.y; acc_s[j][2] = v1.x; acc_s[j][3] = v1.y;
  }
  auto publish_state = [&]() {
    if (!has_state) return;
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
      for (int half = 0; half < 2; half++) {
        uint32_t t[TERMS];
        ck_split(acc_s[j][2 * half], acc_s[j][2 * half + 1], t);
        unsigned char *dst = ck_raw + L::S + (pblk * 16 + g + 8 * half) * L::NROW + ((tw * NT + j) * 8 + 2 * t4) * 2;
#pragma unroll
        for (int i = 0; i < TERMS; i++) *reinterpret_cast<uint32_t *>(dst + i * PB * L::NROW) = t[i];
      }
  };

  stage(0);
  publish_state();
  for (int chunk = 0; chunk < chunks; chunk++) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this chunk's rows and the state terms are there; the other stage is free
    if (L::STAGES == 2 && chunk + 1 < chunks) stage(chunk + 1);
    const uint32_t base = sm + (uint32_t)(chunk % L::STAGES) * L::STAGE;
    const unsigned char *basep = ck_raw + (chunk % L::STAGES) * L::STAGE;
    const float *s_dt = reinterpret_cast<const float *>(basep + L::DT);
    const int r0 = chunk * CQ, n_tok = min(CQ, rows - r0);

    // z of this warp's outputs, asked for now and used at the end of the chunk
    float z[TT][4];
#pragma unroll
    for (int j = 0; j < TT; j++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int t = (tw * TT + j) * 8 + 2 * t4 + (e & 1), p = h * P + p0 + pblk * 16 + g + 8 * (e >> 1);
        z[j][e] = t < n_tok && sh.gated ? proj[(size_t)(r0 + t) * proj_stride + p] : 0.0f;
      }

    // ---- c_t: every warp computes all of them and stores the same values ----
    float c_end;
    {
      const float d0 = s_dt[2 * lane], d1 = s_dt[2 * lane + 1];
      const float v0 = a2 * d0, v1 = a2 * d1;
      float sum = v0 + v1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float u = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += u;
      }
      c_end = __shfl_sync(0xffffffffu, sum, 31);
      const float c1 = sum, c0 = sum - v1;
      s_cum[2 * lane] = c0; s_cum[2 * lane + 1] = c1;
      s_wt[2 * lane] = ck_exp2(c_end - c0) * d0; s_wt[2 * lane + 1] = ck_exp2(c_end - c1) * d1;
      __syncwarp();
    }

    // ---- Xw[s, p] ----
    static_assert(CQ * PB / 8 <= L::THREADS && (CQ * PB / 2) % L::THREADS == 0, "one 16-byte piece of x per thread at most, whole passes over its pairs");
#pragma unroll
    for (int i = 0; i < CQ * PB / 2 / L::THREADS; i++) {
      const int idx = tid + i * L::THREADS, s = idx / (PB / 2), pp = idx % (PB / 2);
      const uint32_t x = *reinterpret_cast<const uint32_t *>(basep + L::X + s * L::PROW + pp * 4);
      const float wt = s_wt[s];
      uint32_t t[TERMS];
      ck_split(__uint_as_float(x << 16) * wt, __uint_as_float(x & 0xffff0000u) * wt, t);
#pragma unroll
      for (int j = 0; j < TERMS; j++) *reinterpret_cast<uint32_t *>(ck_raw + L::XW + (j * CQ + s) * L::PROW + pp * 4) = t[j];
    }

    // ---- G[t, s] = C_t . B_s, weighted by exp(c_t - c_s) dt_s below the diagonal ----
    {
      constexpr int SW = L::WARPS / 4, SC = CQ / SW, ST = SC / 8;  // warps across s, columns and 8-wide tiles of each
      const int tb = warp / SW, s_lo = (warp % SW) * SC;
      const int s_tiles = tb * 16 + 15 >= s_lo ? min(ST, (tb * 16 + 15 - s_lo) / 8 + 1) : 0;  // tiles that are not wholly masked
      float acc[ST][4] = {};
      if (s_tiles > 0) {
#pragma unroll
        for (int k = 0; k < N / 16; k++) {
          uint32_t a[4];
          ck_ldm(a, base + L::C + (tb * 16 + (lane & 15)) * L::NROW + (k * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
          for (int jj = 0; jj < ST / 2; jj++) {
            if (2 * jj < s_tiles) {
              uint32_t b[4];
              ck_ldm(b, base + L::B + (s_lo + jj * 16 + (lane & 7) + 8 * (lane >> 4)) * L::NROW + (k * 16 + ((lane >> 3) & 1) * 8) * 2);
              ck_mma(acc[2 * jj], a, b[0], b[1]);
              ck_mma(acc[2 * jj + 1], a, b[2], b[3]);
            }
          }
        }
      }
      const float ct0 = s_cum[tb * 16 + g], ct1 = s_cum[tb * 16 + g + 8];
#pragma unroll
      for (int j = 0; j < ST; j++) {
        const int s = s_lo + j * 8 + 2 * t4;
        if (j < s_tiles) {
          const float2 cs = *reinterpret_cast<const float2 *>(s_cum + s), ds = *reinterpret_cast<const float2 *>(s_dt + s);
#pragma unroll
          for (int half = 0; half < 2; half++) {
            const int t = tb * 16 + g + 8 * half;
            const float ct = half ? ct1 : ct0;
            const float m0 = s <= t ? acc[j][2 * half] * ck_exp2(ct - cs.x) * ds.x : 0.0f;
            const float m1 = s + 1 <= t ? acc[j][2 * half + 1] * ck_exp2(ct - cs.y) * ds.y : 0.0f;
            uint32_t terms[TERMS];
            ck_split(m0, m1, terms);
#pragma unroll
            for (int i = 0; i < TERMS; i++) *reinterpret_cast<uint32_t *>(ck_raw + L::M + (i * CQ + t) * L::QROW + s * 2) = terms[i];
          }
        } else {
#pragma unroll
          for (int half = 0; half < 2; half++)
#pragma unroll
            for (int i = 0; i < TERMS; i++) *reinterpret_cast<uint32_t *>(ck_raw + L::M + (i * CQ + tb * 16 + g + 8 * half) * L::QROW + s * 2) = 0u;
        }
      }
    }

    // ---- Y^T[p, t] = exp(c_t) S^T C_t ----
    float y[TT][4];
#pragma unroll
    for (int j = 0; j < TT; j++) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.0f;
    if (start_pos > 0 || chunk > 0) {
#pragma unroll
      for (int k = 0; k < N / 16; k++) {
        uint32_t a[TERMS][4];
#pragma unroll
        for (int i = 0; i < TERMS; i++)
          ck_ldm(a[i], sm + L::S + (i * PB + pblk * 16 + (lane & 15)) * L::NROW + (k * 16 + (lane >> 4) * 8) * 2);
        uint32_t b[TT][2];
        ck_load_b<TT>(b, base + L::C + tw * TT * 8 * L::NROW + k * 32, L::NROW, lane);
#pragma unroll
        for (int i = TERMS - 1; i >= 0; i--)
#pragma unroll
          for (int j = 0; j < TT; j++) ck_mma(y[j], a[i], b[j][0], b[j][1]);
      }
#pragma unroll
      for (int j = 0; j < TT; j++) {
        const int t = (tw * TT + j) * 8 + 2 * t4;
        const float e0 = ck_exp2(s_cum[t]), e1 = ck_exp2(s_cum[t + 1]);
        y[j][0] *= e0; y[j][1] *= e1; y[j][2] *= e0; y[j][3] *= e1;
      }
    }
    __syncthreads();  // the weighted products are there, and nobody reads the state terms any more

    // ---- Y^T += X^T G'^T and S^T = exp(c_end) S^T + Xw^T B ----
    const float decay = ck_exp2(c_end);
#pragma unroll
    for (int j = 0; j < NT; j++) { acc_s[j][0] *= decay; acc_s[j][1] *= decay; acc_s[j][2] *= decay; acc_s[j][3] *= decay; }
    const int t_last = (tw * TT + TT) * 8 - 1;  // last token of this warp's Y tile
#pragma unroll
    for (int k = 0; k < CQ / 16; k++) {
      const uint32_t x_off = (k * 16 + (lane & 7) + 8 * (lane >> 4)) * L::PROW + (pblk * 16 + ((lane >> 3) & 1) * 8) * 2;
      if (k * 16 <= t_last) {
        uint32_t x[4];
        ck_ldmt(x, base + L::X + x_off);
#pragma unroll
        for (int i = TERMS - 1; i >= 0; i--) {
          uint32_t b[TT][2];
          ck_load_b<TT>(b, sm + L::M + (i * CQ + tw * TT * 8) * L::QROW + k * 32, L::QROW, lane);
#pragma unroll
          for (int j = 0; j < TT; j++) ck_mma(y[j], x, b[j][0], b[j][1]);
        }
      }
      if (has_state) {
        uint32_t xw[TERMS][4];
#pragma unroll
        for (int i = 0; i < TERMS; i++) ck_ldmt(xw[i], sm + L::XW + i * CQ * L::PROW + x_off);
        if constexpr (NT >= 2) {
          uint32_t b[NT / 2][4];
#pragma unroll
          for (int j = 0; j < NT / 2; j++) ck_ldmt(b[j], base + L::B + (k * 16 + (lane & 15)) * L::NROW + ((tw * NT + 2 * j) * 8 + (lane >> 4) * 8) * 2);
#pragma unroll
          for (int i = TERMS - 1; i >= 0; i--)
#pragma unroll
            for (int j = 0; j < NT / 2; j++) { ck_mma(acc_s[2 * j], xw[i], b[j][0], b[j][1]); ck_mma(acc_s[2 * j + 1], xw[i], b[j][2], b[j][3]); }
        } else {
          uint32_t b0, b1;
          ck_ldmt2(b0, b1, base + L::B + (k * 16 + (lane & 15)) * L::NROW + (tw * NT * 8) * 2);
#pragma unroll
          for (int i = TERMS - 1; i >= 0; i--) ck_mma(acc_s[0], xw[i], b0, b1);
        }
      }
    }
    publish_state();

    // ---- (y + D x) silu(z) ----
#pragma unroll
    for (int j = 0; j < TT; j++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int t = (tw * TT + j) * 8 + 2 * t4 + (e & 1), p = pblk * 16 + g + 8 * (e >> 1);
        if (t < n_tok) {
          const float x = __bfloat162float(*reinterpret_cast<const __nv_bfloat16 *>(basep + L::X + t * L::PROW + p * 2));
          const float v = fmaf(dh, x, y[j][e]);
          out[(size_t)(r0 + t) * inner + h * P + p0 + p] = sh.gated ? v * ck_silu(z[j][e]) : v;
        }
      }
    if (L::STAGES == 1 && chunk + 1 < chunks) {
      __syncthreads();  // nobody reads this chunk's rows any more
      stage(chunk + 1);
    }
  }
  if (has_state)
#pragma unroll
    for (int j = 0; j < NT; j++) {
      *reinterpret_cast<float2 *>(S0 + j * 8) = make_float2(acc_s[j][0], acc_s[j][1]);
      *reinterpret_cast<float2 *>(S0 + 8 * N + j * 8) = make_float2(acc_s[j][2], acc_s[j][3]);
    }
}

template <int N, int PB>
dp_status launch(dp_ctx *ctx, const float *proj, int proj_stride, const __nv_bfloat16 *xbc, const float *dt, const SsmShape &sh, const SsmWeights &w,
                 const SsmState &st, float *out, int rows, const RowMap &map) {
  const int smem = CkLayout<N, PB>::TOTAL;
  static dp_per_device_once attr;
  if (attr.pending(ctx->device)) {
    DP_CUDA(ctx, cudaFuncSetAttribute((ssm_chunk_kernel<N, PB>), cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr.done(ctx->device);
  }
  DP_LAUNCH(ctx, (ssm_chunk_kernel<N, PB>), dim3(sh.heads, sh.vdim / PB), (CkLayout<N, PB>::THREADS), smem, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map.start_pos, map.seq);
  return DP_OK;
}

template <int N>
dp_status pick_cols(dp_ctx *ctx, const float *proj, int proj_stride, const __nv_bfloat16 *xbc, const float *dt, const SsmShape &sh, const SsmWeights &w,
                    const SsmState &st, float *out, int rows, const RowMap &map) {
  // wide column blocks share the C.B products; narrow ones fill the GPU when the heads are few
  if (sh.vdim % 64 == 0 && sh.heads * (sh.vdim / 64) >= ctx->sm_count * 3 / 5) return launch<N, 64>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
  if (sh.vdim % 32 == 0 && sh.heads * (sh.vdim / 32) >= ctx->sm_count * 3 / 5) return launch<N, 32>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
  return launch<N, 16>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
}

}  // namespace

bool dpk_ssm_chunk_ok(const SsmShape &sh, int rows) {
  return rows >= 16 && sh.vdim % 16 == 0 && (sh.state == 32 || sh.state == 64 || sh.state == 128);
}

dp_status dpk_ssm_chunk(dp_ctx *ctx, const float *proj, int proj_stride, const __nv_bfloat16 *xbc, const float *dt, const SsmShape &sh, const SsmWeights &w,
                        const SsmState &st, float *out, int rows, const RowMap &map) {
  switch (sh.state) {
    case 32: return pick_cols<32>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
    case 64: return pick_cols<64>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
    case 128: return pick_cols<128>(ctx, proj, proj_stride, xbc, dt, sh, w, st, out, rows, map);
  }
  return dp_fail(ctx, DP_ERR_UNSUPPORTED, "ssm: state size %d in chunks", sh.state);
}
