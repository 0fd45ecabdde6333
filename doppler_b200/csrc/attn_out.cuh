// Pieces the attention kernels share: which keys a query row sees, and where an output element goes.
#pragma once
#include "common.h"

struct AttnRange { int lo, hi; };

// keys visible to query row qi: [lo, hi) in cache positions
__device__ __forceinline__ AttnRange attn_range(const dpk_attn_params &p, int kv_len, int qi) {
  AttnRange r;
  r.lo = 0;
  r.hi = kv_len;
  const int abs_q = p.start_pos + qi;
  if (p.causal) {
    int lim = abs_q - p.kv_start + 1;  // abs_key <= abs_q
    if (lim < r.hi) r.hi = lim;
  }
  if (p.sliding_window > 0 && abs_q >= p.sliding_window) {
    int first = abs_q - p.sliding_window + 1 - p.kv_start;  // abs_key >= abs_q - window + 1
    if (first > r.lo) r.lo = first;
  }
  if (p.chunk > 0 && r.hi > 0) {
    // the query's own position: given by start_pos under a causal mask, else the last of the sequence's keys
    const int pos = p.causal ? abs_q : r.hi - 1 + p.kv_start;
    const int first = pos / p.chunk * p.chunk - p.kv_start;
    if (first > r.lo) r.lo = first;
  }
  if (r.hi < r.lo) r.hi = r.lo;
  return r;
}

// element d of head h of row z, times the head's output gate where there is one
__device__ __forceinline__ void attn_store(const dpk_attn_params &p, size_t z, int h, int V, int d, float v) {
  if (p.gate) v *= 1.0f / (1.0f + expf(-p.gate[z * p.gate_stride + h]));
  if (p.out_bf16) p.out_bf16[z * p.out_stride + (size_t)h * V + d] = __float2bfloat16_rn(v);
  else p.out[(z * p.num_heads + h) * V + d] = v;
}
