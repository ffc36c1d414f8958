// The part of an engine step that every model shares: packed-batch buffers, pinned staging, page reservation, samplers,
// CUDA graphs of decode-only steps, event timing.  A model (llama.cu, decoder.cu) derives from b200_model and adds its
// weights and its layer stack.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <map>
#include <tuple>
#include <vector>

#include "common.h"
#include "kv_pool.cuh"

b200_status b200_gather_rows(const void* d_src, const int32_t* d_idx, void* d_dst, int32_t rows, int32_t hidden, void* stream);
b200_status b200_scatter_tokens(const uint32_t* d_next, const b200_pack_desc* d_desc, uint32_t* d_last_token, int32_t n_req,
                                const int* d_flags, int flag_a, int flag_b, void* stream);

struct b200_model {
  int vocab = 0, max_rows = 0, max_reqs = 0, max_seqs = 0;
  int max_positions = 0;  // positions a sequence may have, 0: as many as its page table holds
  bool logits_f32 = false;
  bool ready = false;  // every weight is in place
  void* logits = nullptr;  // [max_reqs + extra_rows, vocab], bf16 or f32
  int extra_rows = 0;      // rows beyond the requests' last ones that the buffers hold
  // packed batch
  b200_pack_desc* d_desc = nullptr;
  uint32_t *d_prefill = nullptr, *d_tokens = nullptr, *d_next = nullptr, *d_last_token = nullptr;
  int32_t *d_cu = nullptr, *d_pos = nullptr, *d_row_to_req = nullptr, *d_row_seq = nullptr, *d_row_ctx = nullptr;
  int32_t* d_logit_row = nullptr;  // packed rows whose logits are computed: the requests' last rows, then the wanted ones
  // pinned staging
  b200_pack_desc* h_desc = nullptr;
  uint32_t *h_prefill = nullptr, *h_next = nullptr;
  int32_t* h_state = nullptr;  // [8] pool state words + [2] matmul error words
  std::vector<int32_t> want;   // extra logit rows of the coming step (b200_model_want_logits, used once)
  int last_logit_rows = 0;
  // per-request sampler rows of the coming step (b200_model_set_samplers, used once)
  b200_sample_params *d_samp = nullptr, *h_samp = nullptr;
  float* d_logprobs = nullptr;
  int samp_n = 0;
  bool sampling = false;  // the step in flight samples with d_samp instead of taking the argmax
  int last_n_req = 0;
  long long launches = 0;  // kernels launched by forward calls so far
  // CUDA graphs of decode-only steps, keyed by (requests, device descriptor pointer, the pool's uid, stream, sampling): the
  // first step of a shape runs eagerly (it may grow scratch buffers), the second is captured, later ones replay the graph.
  bool graphs_on = true;
  struct GraphEntry { int seen = 0; cudaGraphExec_t exec = nullptr; long long kernels = 0; };
  std::map<std::tuple<int, const void*, uint64_t, void*, bool>, GraphEntry> graphs;
  // optional CUDA-event timing per category: 0 attention, 1 matmuls, 2 cache append, 3 the rest
  bool prof_on = false;
  std::vector<cudaEvent_t> prof_events;  // pairs
  std::vector<int> prof_cat;
  size_t prof_used = 0;

  virtual ~b200_model();
  // Fails when the pool was built for another model.
  virtual b200_status check_pool(const b200_kv* kv) const = 0;
  // Embedding to logits of the packed batch (T rows; tokens, positions and slots in the buffers above, pages reserved):
  // row i of `logits` belongs to packed row d_logit_row[i], n_logits of them.
  virtual b200_status run_layers(b200_kv* kv, int n_req, int T, int n_logits, void* stream) = 0;
  // Grows the model's own buffers to `rows` logit rows.
  virtual b200_status reserve_logit_rows(int rows) = 0;

  b200_status alloc_step(int vocab, int max_rows, int max_reqs, int max_seqs, bool logits_f32);
  b200_status step(b200_kv* kv, const b200_pack_desc* h_desc, int n_req, const uint32_t* h_prefill_tokens, int n_prefill_tokens,
                   uint32_t* h_next_tokens, int32_t* out_free_pages, void* stream);
  b200_status forward(b200_kv* kv, const b200_pack_desc* d_desc, int n_req, int total_rows, const uint32_t* d_prefill_tokens, void* stream);
  void drop_graphs();
  cudaEvent_t prof_begin(int cat, cudaStream_t s);
  void prof_end(cudaEvent_t e, cudaStream_t s) { if (e) cudaEventRecord(e, s); }

 private:
  b200_status eager(b200_kv* kv, const b200_pack_desc* d_desc, int n_req, int total_rows, const uint32_t* d_prefill_tokens, void* stream);
};

// Runs one call of a step, timed under `cat` when profiling is on (expects `st`, `cs` and a model `m` in scope).
#define MODEL_STEP_CAT(cat, call) \
  do { cudaEvent_t pe_ = m->prof_begin(cat, cs); st = (call); m->prof_end(pe_, cs); if (st != B200_OK) return st; } while (0)
#define MODEL_STEP(call) MODEL_STEP_CAT(3, call)
