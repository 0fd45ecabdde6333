// The decoder runner's state, shared by the two kinds of decoder it schedules: the dense Q4_K decoder (model.cu)
// and decoders described layer by layer (stack.cu).  Sequences, KV allocations, the device-side decode state, the
// step's CUDA graph, the logits and the greedy pick belong to the runner and are the same for both.
#pragma once
#include "common.h"

struct dp_stack;

struct LayerW {
  dp_buf qkv = nullptr, o = nullptr, gateup = nullptr, down = nullptr;
  float *in_norm = nullptr, *post_norm = nullptr, *q_norm = nullptr, *k_norm = nullptr;
};

struct dp_model {
  dp_ctx *ctx;
  dp_model_cfg cfg;
  int nh, nkv, qdim, kvdim, inter, vocab_l, vocab0;  // this rank's share
  int T;                                              // rows of the activation buffers
  std::vector<LayerW> layers;
  dp_buf norms = nullptr, embed = nullptr, lm_head = nullptr;
  float *final_norm = nullptr;
  std::vector<dp_buf> kc, vc;
  dp_buf rope = nullptr;
  float *rope_cos = nullptr, *rope_sin = nullptr;
  dp_buf act = nullptr;  // one slab for all activations
  float *h, *n, *qkv, *q, *att, *gu, *actv, *partial, *logits;
  float *hbuf[3];       // tensor-parallel single-token decode: the residual stream rotates over three buffers (hbuf[0] == h);
                        // a kernel reads one and its CTAs write their shares of the next, so none overwrites what another still reads
  float *h_last;        // where the last forward pass left the hidden state
  unsigned *d_ticket = nullptr;   // device counter of decode steps ever run on this CONTEXT (its exchange area outlives a model):
                                  // hand-off tickets derive from it and never repeat
  dp_buf logits_buf = nullptr;
  dp_buf state = nullptr;  // device ints: pos[B], kvlen[B], tok[B], step, then argmax scratch
  int *d_pos, *d_kvlen, *d_tok, *d_step;
  float *am_vals; int *am_idx; float *am_best; int *am_pair_i; float *am_gather;
  dp_buf out_tokens = nullptr;
  int out_tokens_cap = 0;
  int *pin_state = nullptr;   // page-locked staging of the per-call state block (1024 words) + the status word read back
  int *pin_out = nullptr;     // page-locked staging of the decoded tokens (out_tokens_cap words)
  dp_buf attn_scratch = nullptr;
  dp_buf actq = nullptr;  // fixed-point activation digits of the decode GEMV (sized for the largest K)
  int attn_splits_decode = 1;
  bool recording_decode = false;  // set while a decode step is recorded into its CUDA graph
  bool fuse_qk = true;  // decode: QK norm + RoPE + KV append inside the attention kernel
  std::vector<int> seq_len;
  dp_graph *graph[2] = {nullptr, nullptr};
  int graph_batch[2] = {0, 0};
  cudaEvent_t ev0 = nullptr, ev1 = nullptr;
  double last_ms = 0;
  size_t weight_bytes = 0;
  int allreduce_mode = 0;
  dp_stack *stack = nullptr;  // a decoder described layer by layer (stack.cu): its weights, sequence state and activations
  bool final_norm_done = false;  // set by run_layers when the exchange kernel already applied the final RMSNorm
};

// model.cu: device state of the decode loop, logits, argmax scratch and events (needs m->cfg, m->vocab_l, m->T)
dp_status dp_model_alloc_runner(dp_model *m);

// stack.cu
void dp_stack_destroy(dp_model *m);
dp_status dp_stack_ready(dp_model *m);  // every tensor loaded
dp_status dp_stack_embed(dp_model *m, const int *ids, int rows, bool decode);
dp_status dp_stack_run_layers(dp_model *m, int rows, bool decode, int seq, int start_pos);
dp_status dp_stack_logits(dp_model *m, const float *hrow, int rows);
