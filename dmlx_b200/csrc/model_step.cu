// Engine step of any model over a packed ragged batch: pack -> page reservation -> the model's layer stack -> sampling,
// all on one stream (the greedy branch of generateBatchStep, src/generation.zig:104-145, and SamplerConfig.sample where
// sampler rows were set).
#include "model_step.cuh"

#include <algorithm>
#include <cstring>

#include "qmm.cuh"

b200_model::~b200_model() {
  void* dev[] = {logits, d_desc, d_prefill, d_tokens, d_next, d_last_token, d_cu, d_pos, d_row_to_req, d_row_seq, d_row_ctx, d_logit_row,
                 d_samp, d_logprobs};
  for (void* p : dev) if (p) cudaFree(p);
  if (h_desc) cudaFreeHost(h_desc);
  if (h_prefill) cudaFreeHost(h_prefill);
  if (h_next) cudaFreeHost(h_next);
  if (h_samp) cudaFreeHost(h_samp);
  if (h_state) cudaFreeHost(h_state);
  for (cudaEvent_t e : prof_events) cudaEventDestroy(e);
  for (auto& g : graphs) if (g.second.exec) cudaGraphExecDestroy(g.second.exec);
}

b200_status b200_model::alloc_step(int vocab_, int max_rows_, int max_reqs_, int max_seqs_, bool f32) {
  vocab = vocab_; max_rows = max_rows_; max_reqs = max_reqs_; max_seqs = max_seqs_; logits_f32 = f32;
  const int R = max_rows, Q = max_reqs;
  auto dev = [](auto** p, size_t bytes) { return cudaMalloc((void**)p, bytes) == cudaSuccess; };
  auto pin = [](auto** p, size_t bytes) { return cudaMallocHost((void**)p, bytes) == cudaSuccess; };
  if (!dev(&logits, (size_t)Q * vocab * (f32 ? 4 : 2)) || !dev(&d_desc, sizeof(b200_pack_desc) * Q) || !dev(&d_prefill, sizeof(uint32_t) * R) ||
      !dev(&d_tokens, sizeof(uint32_t) * R) || !dev(&d_next, sizeof(uint32_t) * Q) || !dev(&d_last_token, sizeof(uint32_t) * max_seqs) ||
      !dev(&d_cu, sizeof(int32_t) * (Q + 1)) || !dev(&d_pos, sizeof(int32_t) * R) || !dev(&d_row_to_req, sizeof(int32_t) * R) ||
      !dev(&d_row_seq, sizeof(int32_t) * R) || !dev(&d_row_ctx, sizeof(int32_t) * R) || !dev(&d_logit_row, sizeof(int32_t) * Q) ||
      !dev(&d_samp, sizeof(b200_sample_params) * Q) || !dev(&d_logprobs, sizeof(float) * Q)) {
    b200_set_error("model: device allocation of the step buffers failed");
    return B200_ERR_CUDA;
  }
  if (!pin(&h_desc, sizeof(b200_pack_desc) * Q) || !pin(&h_prefill, sizeof(uint32_t) * R) || !pin(&h_next, sizeof(uint32_t) * Q) ||
      !pin(&h_samp, sizeof(b200_sample_params) * Q) || !pin(&h_state, sizeof(int32_t) * 16)) {
    b200_set_error("pinned host allocation failed");
    return B200_ERR_CUDA;
  }
  B200_CUDA_TRY(cudaMemset(d_last_token, 0, sizeof(uint32_t) * max_seqs));
  return B200_OK;
}

cudaEvent_t b200_model::prof_begin(int cat, cudaStream_t s) {
  if (!prof_on) return nullptr;
  if (prof_used + 2 > prof_events.size()) {
    cudaEvent_t a, b;
    cudaEventCreate(&a);
    cudaEventCreate(&b);
    prof_events.push_back(a);
    prof_events.push_back(b);
    prof_cat.push_back(cat);
  }
  prof_cat[prof_used / 2] = cat;
  cudaEventRecord(prof_events[prof_used], s);
  prof_used += 2;
  return prof_events[prof_used - 1];
}

void b200_model::drop_graphs() {
  for (auto& g : graphs)
    if (g.second.exec) { cudaGraphExecDestroy(g.second.exec); g.second.exec = nullptr; g.second.seen = 0; }
}

b200_status b200_model::forward(b200_kv* kv, const b200_pack_desc* desc, int n_req, int total_rows, const uint32_t* d_prefill_tokens,
                                void* stream) {
  // Decode-only steps (one row per request) are launch-bound at small batch: replay them as a graph.
  // (the legacy default stream cannot be captured)
  if (!graphs_on || prof_on || total_rows != n_req || n_req <= 0 || !ready || stream == nullptr || !want.empty())
    return eager(kv, desc, n_req, total_rows, d_prefill_tokens, stream);
  auto& ge = graphs[std::make_tuple((int)n_req, (const void*)desc, kv->uid, stream, sampling)];
  ge.seen += 1;
  if (ge.seen == 1) return eager(kv, desc, n_req, total_rows, d_prefill_tokens, stream);
  cudaStream_t cs = (cudaStream_t)stream;
  if (!ge.exec) {
    if (graphs.size() > 64) {  // bounded cache: drop everything else
      for (auto& kvp : graphs) if (kvp.second.exec && &kvp.second != &ge) { cudaGraphExecDestroy(kvp.second.exec); kvp.second.exec = nullptr; kvp.second.seen = 0; }
    }
    cudaGraph_t graph = nullptr;
    B200_CUDA_TRY(cudaStreamBeginCapture(cs, cudaStreamCaptureModeThreadLocal));
    const long long before = launches;
    b200_status st = eager(kv, desc, n_req, total_rows, d_prefill_tokens, stream);
    ge.kernels = launches - before;  // nodes of the graph
    launches = before;
    cudaError_t e = cudaStreamEndCapture(cs, &graph);
    if (st != B200_OK) { if (graph) cudaGraphDestroy(graph); return st; }
    if (e != cudaSuccess) { b200_set_error("graph capture failed: %s", cudaGetErrorString(e)); cudaGetLastError(); return B200_ERR_CUDA; }
    e = cudaGraphInstantiate(&ge.exec, graph, 0);
    cudaGraphDestroy(graph);
    if (e != cudaSuccess) { ge.exec = nullptr; b200_set_error("graph instantiate failed: %s", cudaGetErrorString(e)); return B200_ERR_CUDA; }
  }
  B200_CUDA_TRY(cudaGraphLaunch(ge.exec, cs));
  last_n_req = last_logit_rows = n_req;
  launches += ge.kernels;
  return B200_OK;
}

b200_status b200_model::eager(b200_kv* kv, const b200_pack_desc* desc, int n_req, int total_rows, const uint32_t* d_prefill_tokens,
                              void* stream) {
  b200_model* m = this;
  if (!ready) { b200_set_error("model: weights not finalized"); return B200_ERR_INVALID_ARGUMENT; }
  if (n_req < 0 || n_req > max_reqs || total_rows < 0 || total_rows > max_rows) {
    b200_set_error("model: %d requests / %d rows exceed the configured %d / %d", n_req, total_rows, max_reqs, max_rows);
    return B200_ERR_CAPACITY;
  }
  b200_status st = check_pool(kv);
  if (st != B200_OK) return st;
  const int n_logits = n_req + (int)want.size();
  last_n_req = n_req;
  last_logit_rows = n_logits;
  if (n_req == 0 || total_rows == 0) return B200_OK;
  const long long launches_before = g_b200_launch_counter;
  cudaStream_t cs = (cudaStream_t)stream;
  MODEL_STEP(b200_pack_batch(desc, n_req, d_prefill_tokens, d_last_token, d_cu, d_tokens, d_pos, d_row_to_req, d_row_seq, d_row_ctx,
                             d_logit_row, total_rows, stream));
  if (!want.empty())
    B200_CUDA_TRY(cudaMemcpyAsync(d_logit_row + n_req, want.data(), sizeof(int32_t) * want.size(), cudaMemcpyHostToDevice, cs));
  MODEL_STEP(b200_kv_reserve(kv, desc, n_req, stream));
  st = run_layers(kv, n_req, total_rows, n_logits, stream);
  if (st != B200_OK) return st;
  if (sampling) {
    MODEL_STEP(b200_sample_rows(logits, logits_f32 ? 1 : 0, n_req, vocab, d_samp, nullptr, nullptr, nullptr, d_next, d_logprobs, stream));
  } else if (logits_f32) {
    MODEL_STEP(b200_argmax_f32((const float*)logits, n_req, vocab, d_next, stream));
  } else {
    MODEL_STEP(b200_argmax(logits, n_req, vocab, d_next, stream));
  }
  MODEL_STEP(b200_scatter_tokens(d_next, desc, d_last_token, n_req, kv->dev.state, ST_ERR, ST_ATTN_ERR, stream));
  launches += g_b200_launch_counter - launches_before;
  return B200_OK;
}

b200_status b200_model::step(b200_kv* kv, const b200_pack_desc* descs, int n_req, const uint32_t* h_prefill_tokens, int n_prefill_tokens,
                             uint32_t* h_next_tokens, int32_t* out_free_pages, void* stream) {
  struct ClearWant {  // the wanted rows and sampler rows belong to this step, whatever becomes of it
    b200_model* m;
    ~ClearWant() { m->want.clear(); m->samp_n = 0; m->sampling = false; }
  } clear{this};
  if (n_req < 0 || n_req > max_reqs || n_prefill_tokens < 0 || n_prefill_tokens > max_rows) {
    b200_set_error("model step: %d requests / %d prefill tokens exceed the configured limits", n_req, n_prefill_tokens);
    return B200_ERR_CAPACITY;
  }
  cudaStream_t s = (cudaStream_t)stream;
  long long total = 0;
  for (int i = 0; i < n_req; ++i) {
    h_desc[i] = descs[i];
    total += descs[i].count > 0 ? descs[i].count : 0;
  }
  if (total > max_rows) { b200_set_error("model step: %lld rows > max_rows %d", total, max_rows); return B200_ERR_CAPACITY; }
  // positions beyond a page table would be read from the next sequence's
  long long most = (long long)kv->cfg.max_pages_per_seq * kv->cfg.page_size;
  if (max_positions > 0) most = std::min<long long>(most, max_positions);
  for (int i = 0; i < n_req; ++i)
    if (descs[i].base_pos < 0 || (long long)descs[i].base_pos + std::max(descs[i].count, 0) > most) {
      b200_set_error("model step: positions %d + %d exceed the %lld a sequence may have", descs[i].base_pos, descs[i].count, most);
      return B200_ERR_INVALID_BATCH_INDEX;
    }
  for (int32_t r : want)
    if (r < 0 || r >= total) { b200_set_error("model step: logits of row %d wanted, the step has %lld", r, total); return B200_ERR_INVALID_ARGUMENT; }
  for (int i = 0; i < n_prefill_tokens; ++i)
    if (h_prefill_tokens[i] >= (uint32_t)vocab) {
      b200_set_error("model step: token %u outside the vocabulary of %d", h_prefill_tokens[i], vocab);
      return B200_ERR_INVALID_ARGUMENT;
    }
  if (n_prefill_tokens > 0) std::memcpy(h_prefill, h_prefill_tokens, sizeof(uint32_t) * n_prefill_tokens);
  if (n_req > 0) B200_CUDA_TRY(cudaMemcpyAsync(d_desc, h_desc, sizeof(b200_pack_desc) * n_req, cudaMemcpyHostToDevice, s));
  if (n_prefill_tokens > 0)
    B200_CUDA_TRY(cudaMemcpyAsync(d_prefill, h_prefill, sizeof(uint32_t) * n_prefill_tokens, cudaMemcpyHostToDevice, s));
  sampling = samp_n > 0;
  if (sampling) {
    if (samp_n != n_req) {
      b200_set_error("model step: %d sampler rows for %d requests", samp_n, n_req);
      return B200_ERR_INVALID_ARGUMENT;
    }
    B200_CUDA_TRY(cudaMemcpyAsync(d_samp, h_samp, sizeof(b200_sample_params) * n_req, cudaMemcpyHostToDevice, s));
  }
  b200_status st = forward(kv, d_desc, n_req, (int)total, d_prefill, stream);
  if (st != B200_OK) return st;
  if (n_req > 0) B200_CUDA_TRY(cudaMemcpyAsync(h_next, d_next, sizeof(uint32_t) * n_req, cudaMemcpyDeviceToHost, s));
  B200_CUDA_TRY(cudaMemcpyAsync(h_state, kv->dev.state, sizeof(int32_t) * 8, cudaMemcpyDeviceToHost, s));
  st = b200_qmm_error_words_async(h_state + 8, stream);
  if (st != B200_OK) return st;
  B200_CUDA_TRY(cudaStreamSynchronize(s));
  for (int i = 0; i < n_req; ++i) h_next_tokens[i] = h_next[i];
  if (out_free_pages) *out_free_pages = h_state[ST_FREE_TOP];
  if (h_state[8] == 0) h_state[8] = h_state[9];
  if (h_state[ST_ERR] != 0 || h_state[ST_ATTN_ERR] != 0 || h_state[8] != 0) {
    int32_t word = 0;
    b200_kv_error_word(kv, &word);  // clears the pool's words
    int32_t q = 0;
    b200_qmm_error_word(&q);
    const int code = h_state[ST_ERR] ? h_state[ST_ERR] : (h_state[ST_ATTN_ERR] ? h_state[ST_ATTN_ERR] : h_state[8]);
    b200_set_error("model step: a kernel flagged %s", b200_status_name(code));
    return code;
  }
  return B200_OK;
}

extern "C" {

void b200_model_get_info(const b200_model* m, b200_model_info* out) {
  *out = b200_model_info{m->vocab, m->max_rows, m->max_reqs, m->max_seqs, m->logits_f32 ? 1 : 0, m->max_positions};
}

b200_status b200_model_step(b200_model* m, b200_kv* kv, const b200_pack_desc* h_desc, int32_t n_req, const uint32_t* h_prefill_tokens,
                            int32_t n_prefill_tokens, uint32_t* h_next_tokens, int32_t* out_free_pages, void* stream) {
  return m->step(kv, h_desc, n_req, h_prefill_tokens, n_prefill_tokens, h_next_tokens, out_free_pages, stream);
}

b200_status b200_model_forward(b200_model* m, b200_kv* kv, const b200_pack_desc* d_desc, int32_t n_req, int32_t total_rows,
                               const uint32_t* d_prefill_tokens, void* stream) {
  return m->forward(kv, d_desc, n_req, total_rows, d_prefill_tokens, stream);
}

// Device buffers the caller may use for a device-resident step (benchmarks): descriptor array
// [max_reqs], prefill token buffer [max_rows], next-token output [max_reqs].
void b200_model_device_buffers(b200_model* m, b200_pack_desc** d_desc, uint32_t** d_prefill, uint32_t** d_next) {
  if (d_desc) *d_desc = m->d_desc;
  if (d_prefill) *d_prefill = m->d_prefill;
  if (d_next) *d_next = m->d_next;
}

b200_status b200_model_set_samplers(b200_model* m, const b200_sample_params* h_rows, int32_t n_req) {
  if (n_req < 0 || n_req > m->max_reqs || (n_req > 0 && h_rows == nullptr)) {
    b200_set_error("set_samplers: %d rows (the model holds %d requests)", n_req, m->max_reqs);
    return B200_ERR_INVALID_ARGUMENT;
  }
  for (int i = 0; i < n_req; ++i) m->h_samp[i] = h_rows[i];
  m->samp_n = n_req;
  return B200_OK;
}

b200_status b200_model_last_logprobs(b200_model* m, float* h_out, int32_t n_req) {
  if (n_req > m->last_n_req) { b200_set_error("last_logprobs: %d rows requested, last step had %d", n_req, m->last_n_req); return B200_ERR_CAPACITY; }
  if (n_req > 0) B200_CUDA_TRY(cudaMemcpy(h_out, m->d_logprobs, sizeof(float) * n_req, cudaMemcpyDeviceToHost));
  return B200_OK;
}

b200_status b200_model_want_logits(b200_model* m, const int32_t* h_rows, int32_t n) {
  if (n < 0 || (n > 0 && !h_rows)) { b200_set_error("want_logits: %d rows", n); return B200_ERR_INVALID_ARGUMENT; }
  if (n > m->extra_rows) {
    const int extra = std::max(n, 2 * m->extra_rows), rows = m->max_reqs + extra;
    void* lg = nullptr;
    int32_t* lr = nullptr;
    B200_CUDA_TRY(cudaDeviceSynchronize());
    b200_status st = m->reserve_logit_rows(rows);
    if (st != B200_OK) return st;
    if (cudaMalloc(&lg, (size_t)rows * m->vocab * (m->logits_f32 ? 4 : 2)) != cudaSuccess ||
        cudaMalloc((void**)&lr, sizeof(int32_t) * rows) != cudaSuccess) {
      if (lg) cudaFree(lg);
      b200_set_error("want_logits: no memory for %d rows of logits", rows);
      return B200_ERR_CUDA;
    }
    cudaFree(m->logits);
    cudaFree(m->d_logit_row);
    m->logits = lg;
    m->d_logit_row = lr;
    m->extra_rows = extra;
    m->drop_graphs();  // they hold the old buffers
  }
  m->want.assign(h_rows, h_rows + n);
  return B200_OK;
}

b200_status b200_model_logits(b200_model* m, int32_t first, int32_t n, float* h_out) {
  if (first < 0 || n < 0 || first + n > m->last_logit_rows) {
    b200_set_error("logits: rows %d..%d requested, the last step computed %d", first, first + n, m->last_logit_rows);
    return B200_ERR_CAPACITY;
  }
  const size_t count = (size_t)n * m->vocab, off = (size_t)first * m->vocab;
  if (count == 0) return B200_OK;
  if (m->logits_f32) {
    B200_CUDA_TRY(cudaMemcpy(h_out, (const float*)m->logits + off, count * 4, cudaMemcpyDeviceToHost));
    return B200_OK;
  }
  std::vector<uint16_t> bits(count);
  B200_CUDA_TRY(cudaMemcpy(bits.data(), (const uint16_t*)m->logits + off, count * 2, cudaMemcpyDeviceToHost));
  for (size_t i = 0; i < count; ++i) {
    const uint32_t u = (uint32_t)bits[i] << 16;
    std::memcpy(h_out + i, &u, 4);
  }
  return B200_OK;
}

int64_t b200_model_launch_count(const b200_model* m) { return m->launches; }
void b200_model_enable_graphs(b200_model* m, int32_t on) { m->graphs_on = on != 0; }

// CUDA-event timing of the step's kernels by category (0 attention, 1 matmuls, 2 cache append,
// 3 the rest).  collect() synchronises the device, adds the elapsed time of every recorded call
// to ms[4] / calls[4] and clears the record.
void b200_model_profile_enable(b200_model* m, int32_t on) { m->prof_on = on != 0; m->prof_used = 0; }
b200_status b200_model_profile_collect(b200_model* m, double* ms, int64_t* calls) {
  B200_CUDA_TRY(cudaDeviceSynchronize());
  for (int i = 0; i < 4; ++i) { ms[i] = 0; calls[i] = 0; }
  for (size_t i = 0; i + 1 < m->prof_used; i += 2) {
    float t = 0.f;
    B200_CUDA_TRY(cudaEventElapsedTime(&t, m->prof_events[i], m->prof_events[i + 1]));
    ms[m->prof_cat[i / 2]] += t;
    calls[m->prof_cat[i / 2]] += 1;
  }
  m->prof_used = 0;
  return B200_OK;
}

}  // extern "C"
