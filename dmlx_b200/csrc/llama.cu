// LLaMA-architecture layer stack over a packed ragged batch (model_step.cu packs it and reserves its pages): embed -> N x (RMSNorm, fused QKV matmul, RoPE, paged KV append,
// paged attention, output matmul + residual, RMSNorm, gate/up matmul + SwiGLU, down matmul +
// residual) -> last-row gather -> RMSNorm -> lm_head, all on one stream.
// Follows LlamaModel.forward / LlamaTransformerBlock.forward / LlamaAttention.forward /
// LlamaMLP.forward (src/models/llama.zig:556-609, 460-481, 138-299, 372-438) and the greedy branch
// of generateBatchStep (src/generation.zig:104-145); per-row positions replace the reference's
// scalar RoPE offset, and attention reads the page pool in place instead of a gathered copy.
#include <cuda_bf16.h>

#include <cstring>
#include <map>
#include <vector>

#include "common.h"
#include "kv_pool.cuh"
#include "model_step.cuh"
#include "qmm.cuh"

namespace {
struct HostMat {
  int mode = -1, n = 0, k = 0;
  std::vector<unsigned char> packed, scales, biases;
};
size_t packed_row_bytes(int mode, int k) { return mode == B200_Q_AFFINE4_G64 ? (size_t)k / 2 : (mode == B200_Q_MXFP4_G32 ? (size_t)k / 2 : (size_t)k * 2); }
size_t scale_row_bytes(int mode, int k) { return mode == B200_Q_AFFINE4_G64 ? (size_t)k / 64 * 2 : (mode == B200_Q_MXFP4_G32 ? (size_t)k / 32 : 0); }
}  // namespace

struct b200_llama : b200_model {
  b200_llama_config cfg{};
  std::map<std::pair<int, int>, HostMat> staged;
  __nv_bfloat16* embed = nullptr;
  std::vector<__nv_bfloat16*> attn_norm, ffn_norm;
  __nv_bfloat16* final_norm = nullptr;
  std::vector<b200_qweight*> wqkv, wo, wgu, wdown;
  b200_qweight* lm_head = nullptr;
  // activations
  __nv_bfloat16 *x = nullptr, *h = nullptr, *qkv = nullptr, *attn = nullptr, *act = nullptr, *last_h = nullptr, *last_hn = nullptr;
  bool fuse_qkv_rope = true;  // b200_llama_set_fused_qkv_rope

  ~b200_llama() override;
  b200_status check_pool(const b200_kv* kv) const override;
  b200_status run_layers(b200_kv* kv, int n_req, int T, int n_logits, void* stream) override;
  b200_status reserve_logit_rows(int rows) override;
};


#define L_ALLOC(ptr, bytes)                                                                            \
  do {                                                                                                 \
    cudaError_t e_ = cudaMalloc((void**)&(ptr), (bytes));                                              \
    if (e_ != cudaSuccess) {                                                                           \
      b200_set_error("cudaMalloc(%zu) failed: %s", (size_t)(bytes), cudaGetErrorString(e_));           \
      b200_llama_destroy(m);                                                                           \
      return B200_ERR_CUDA;                                                                            \
    }                                                                                                  \
  } while (0)

extern "C" {

b200_status b200_llama_create(const b200_llama_config* c, b200_llama** out) {
  *out = nullptr;
  b200_status st = b200_require_device();
  if (st != B200_OK) return st;
  if (c->n_layers <= 0 || c->hidden % 64 != 0 || c->ffn % 64 != 0 || (c->n_heads * c->head_dim) % 64 != 0 ||
      c->n_heads % c->n_kv_heads != 0 || c->max_rows <= 0 || c->max_reqs <= 0 || c->vocab <= 0) {
    b200_set_error("llama: invalid configuration (hidden, ffn and heads*head_dim must be multiples of 64)");
    return B200_ERR_INVALID_ARGUMENT;
  }
  auto* m = new b200_llama();
  m->cfg = *c;
  const int L = c->n_layers, R = c->max_rows, Q = c->max_reqs;
  const size_t qkv_dim = (size_t)(c->n_heads + 2 * c->n_kv_heads) * c->head_dim;
  m->attn_norm.assign(L, nullptr); m->ffn_norm.assign(L, nullptr);
  m->wqkv.assign(L, nullptr); m->wo.assign(L, nullptr); m->wgu.assign(L, nullptr); m->wdown.assign(L, nullptr);
  L_ALLOC(m->embed, (size_t)c->vocab * c->hidden * 2);
  for (int l = 0; l < L; ++l) { L_ALLOC(m->attn_norm[l], (size_t)c->hidden * 2); L_ALLOC(m->ffn_norm[l], (size_t)c->hidden * 2); }
  L_ALLOC(m->final_norm, (size_t)c->hidden * 2);
  L_ALLOC(m->x, (size_t)R * c->hidden * 2);
  L_ALLOC(m->h, (size_t)R * c->hidden * 2);
  L_ALLOC(m->qkv, (size_t)R * qkv_dim * 2);
  L_ALLOC(m->attn, (size_t)R * c->n_heads * c->head_dim * 2);
  L_ALLOC(m->act, (size_t)R * c->ffn * 2);
  L_ALLOC(m->last_h, (size_t)Q * c->hidden * 2);
  L_ALLOC(m->last_hn, (size_t)Q * c->hidden * 2);
  st = m->alloc_step(c->vocab, R, Q, c->max_seqs, false);
  if (st != B200_OK) { b200_llama_destroy(m); return st; }
  *out = m;
  return B200_OK;
}

void b200_llama_destroy(b200_llama* m) { delete m; }
b200_model* b200_llama_model(b200_llama* m) { return m; }

static bool linear_dims(const b200_llama_config& c, int which, int* n, int* k) {
  const int qd = c.n_heads * c.head_dim, kd = c.n_kv_heads * c.head_dim;
  switch (which) {
    case B200_W_Q: *n = qd; *k = c.hidden; return true;
    case B200_W_K: case B200_W_V: *n = kd; *k = c.hidden; return true;
    case B200_W_O: *n = c.hidden; *k = qd; return true;
    case B200_W_GATE: case B200_W_UP: *n = c.ffn; *k = c.hidden; return true;
    case B200_W_DOWN: *n = c.hidden; *k = c.ffn; return true;
    case B200_W_LM_HEAD: *n = c.vocab; *k = c.hidden; return true;
    default: return false;
  }
}

b200_status b200_llama_set_linear(b200_llama* m, int32_t layer, int32_t which, int32_t mode, const void* h_packed,
                                  const void* h_scales, const void* h_biases) {
  int n = 0, k = 0;
  if (!linear_dims(m->cfg, which, &n, &k) || (which != B200_W_LM_HEAD && (layer < 0 || layer >= m->cfg.n_layers))) {
    b200_set_error("set_linear: bad layer/which (%d/%d)", layer, which);
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (mode < 0 || mode > B200_Q_BF16) { b200_set_error("set_linear: unknown mode %d", mode); return B200_ERR_INVALID_QUANT_BITS; }
  HostMat hm;
  hm.mode = mode; hm.n = n; hm.k = k;
  const size_t pb = packed_row_bytes(mode, k) * n, sb = scale_row_bytes(mode, k) * n;
  hm.packed.assign((const unsigned char*)h_packed, (const unsigned char*)h_packed + pb);
  if (sb) hm.scales.assign((const unsigned char*)h_scales, (const unsigned char*)h_scales + sb);
  if (mode == B200_Q_AFFINE4_G64) hm.biases.assign((const unsigned char*)h_biases, (const unsigned char*)h_biases + sb);
  m->staged[{which == B200_W_LM_HEAD ? -1 : layer, which}] = std::move(hm);
  return B200_OK;
}

b200_status b200_llama_set_embedding(b200_llama* m, const void* h_bf16) {
  B200_CUDA_TRY(cudaMemcpy(m->embed, h_bf16, (size_t)m->cfg.vocab * m->cfg.hidden * 2, cudaMemcpyHostToDevice));
  return B200_OK;
}

b200_status b200_llama_set_norm(b200_llama* m, int32_t layer, int32_t which, const void* h_bf16) {
  __nv_bfloat16* dst = layer < 0 ? m->final_norm : (which == 0 ? m->attn_norm[layer] : m->ffn_norm[layer]);
  if (layer >= m->cfg.n_layers) { b200_set_error("set_norm: layer out of range"); return B200_ERR_INVALID_ARGUMENT; }
  B200_CUDA_TRY(cudaMemcpy(dst, h_bf16, (size_t)m->cfg.hidden * 2, cudaMemcpyHostToDevice));
  return B200_OK;
}

// Row-wise concatenation (and optional interleave) of staged matrices into one weight.
static b200_status fuse(b200_llama* m, int layer, const std::vector<int>& which, bool interleave, b200_qweight** out) {
  std::vector<const HostMat*> parts;
  for (int w : which) {
    auto it = m->staged.find({layer, w});
    if (it == m->staged.end()) { b200_set_error("finalize: weight %d of layer %d was never set", w, layer); return B200_ERR_INVALID_ARGUMENT; }
    parts.push_back(&it->second);
  }
  const int mode = parts[0]->mode, k = parts[0]->k;
  int n = 0;
  for (auto* p : parts) {
    if (p->mode != mode || p->k != k) { b200_set_error("finalize: fused weights must share mode and K"); return B200_ERR_INVALID_ARGUMENT; }
    n += p->n;
  }
  const size_t prb = packed_row_bytes(mode, k), srb = scale_row_bytes(mode, k);
  std::vector<unsigned char> packed(prb * n), scales(srb * n), biases(mode == B200_Q_AFFINE4_G64 ? srb * n : 0);
  int row = 0;
  auto put = [&](const HostMat* p, int r) {
    std::memcpy(&packed[prb * row], &p->packed[prb * r], prb);
    if (srb) std::memcpy(&scales[srb * row], &p->scales[srb * r], srb);
    if (!biases.empty()) std::memcpy(&biases[srb * row], &p->biases[srb * r], srb);
    ++row;
  };
  if (interleave) {
    for (int r = 0; r < parts[0]->n; ++r) for (auto* p : parts) put(p, r);
  } else {
    for (auto* p : parts) for (int r = 0; r < p->n; ++r) put(p, r);
  }
  b200_status st = b200_qweight_create(mode, 1, n, k, packed.data(), scales.empty() ? nullptr : scales.data(),
                                       biases.empty() ? nullptr : biases.data(), out);
  if (st == B200_OK) for (int w : which) m->staged.erase({layer, w});
  return st;
}

b200_status b200_llama_finalize(b200_llama* m) {
  for (int l = 0; l < m->cfg.n_layers; ++l) {
    b200_status st;
    if ((st = fuse(m, l, {B200_W_Q, B200_W_K, B200_W_V}, false, &m->wqkv[l])) != B200_OK) return st;
    if ((st = fuse(m, l, {B200_W_O}, false, &m->wo[l])) != B200_OK) return st;
    if ((st = fuse(m, l, {B200_W_GATE, B200_W_UP}, true, &m->wgu[l])) != B200_OK) return st;
    if ((st = fuse(m, l, {B200_W_DOWN}, false, &m->wdown[l])) != B200_OK) return st;
  }
  b200_status st = fuse(m, -1, {B200_W_LM_HEAD}, false, &m->lm_head);
  if (st != B200_OK) return st;
  m->ready = true;
  return B200_OK;
}

// Synthetic model for benchmarks: every matrix generated on the device, norm weights 1,
// embedding small random values.
b200_status b200_llama_random_init(b200_llama* m, int32_t mode, uint32_t seed) {
  const b200_llama_config& c = m->cfg;
  const int qkv_n = (c.n_heads + 2 * c.n_kv_heads) * c.head_dim;
  if (qkv_n % 128 || c.hidden % 128 || c.ffn % 64 || c.vocab % 128) {
    b200_set_error("random_init: projection sizes must be multiples of 128");
    return B200_ERR_INVALID_ARGUMENT;
  }
  b200_status st;
  for (int l = 0; l < c.n_layers; ++l) {
    if ((st = b200_qweight_random(mode, 1, qkv_n, c.hidden, seed + 16 * l + 1, &m->wqkv[l])) != B200_OK) return st;
    if ((st = b200_qweight_random(mode, 1, c.hidden, c.n_heads * c.head_dim, seed + 16 * l + 2, &m->wo[l])) != B200_OK) return st;
    if ((st = b200_qweight_random(mode, 1, 2 * c.ffn, c.hidden, seed + 16 * l + 3, &m->wgu[l])) != B200_OK) return st;
    if ((st = b200_qweight_random(mode, 1, c.hidden, c.ffn, seed + 16 * l + 4, &m->wdown[l])) != B200_OK) return st;
  }
  if ((st = b200_qweight_random(mode, 1, c.vocab, c.hidden, seed + 7, &m->lm_head)) != B200_OK) return st;
  std::vector<uint16_t> ones(c.hidden, 0x3F80);
  for (int l = 0; l < c.n_layers; ++l) {
    B200_CUDA_TRY(cudaMemcpy(m->attn_norm[l], ones.data(), c.hidden * 2, cudaMemcpyHostToDevice));
    B200_CUDA_TRY(cudaMemcpy(m->ffn_norm[l], ones.data(), c.hidden * 2, cudaMemcpyHostToDevice));
  }
  B200_CUDA_TRY(cudaMemcpy(m->final_norm, ones.data(), c.hidden * 2, cudaMemcpyHostToDevice));
  b200_qweight* tmp = nullptr;  // reuse the dense random generator for the embedding table
  std::vector<uint16_t> emb((size_t)c.vocab * c.hidden);
  uint32_t s = seed * 2654435761u + 12345u;
  for (auto& e : emb) { s = s * 1664525u + 1013904223u; e = (uint16_t)(((s >> 16) & 0x807F) | 0x3C80); }
  (void)tmp;
  B200_CUDA_TRY(cudaMemcpy(m->embed, emb.data(), emb.size() * 2, cudaMemcpyHostToDevice));
  m->ready = true;
  return B200_OK;
}

}  // extern "C"

b200_llama::~b200_llama() {
  void* dev[] = {embed, final_norm, x, h, qkv, attn, act, last_h, last_hn};
  for (void* p : dev) if (p) cudaFree(p);
  for (auto* p : attn_norm) if (p) cudaFree(p);
  for (auto* p : ffn_norm) if (p) cudaFree(p);
  for (auto* w : wqkv) b200_qweight_destroy(w);
  for (auto* w : wo) b200_qweight_destroy(w);
  for (auto* w : wgu) b200_qweight_destroy(w);
  for (auto* w : wdown) b200_qweight_destroy(w);
  b200_qweight_destroy(lm_head);
}

b200_status b200_llama::check_pool(const b200_kv* kv) const {
  if (kv->layered || kv->cfg.n_layers != cfg.n_layers || kv->cfg.n_kv_heads != cfg.n_kv_heads || kv->cfg.head_dim != cfg.head_dim ||
      kv->cfg.n_q_heads != cfg.n_heads) {
    b200_set_error("llama: the page pool was built for a different model shape");
    return B200_ERR_INVALID_ARGUMENT;
  }
  return B200_OK;
}

b200_status b200_llama::reserve_logit_rows(int rows) {
  __nv_bfloat16 *a = nullptr, *b = nullptr;
  if (cudaMalloc((void**)&a, (size_t)rows * cfg.hidden * 2) != cudaSuccess || cudaMalloc((void**)&b, (size_t)rows * cfg.hidden * 2) != cudaSuccess) {
    if (a) cudaFree(a);
    b200_set_error("llama: no memory for %d logit rows", rows);
    return B200_ERR_CUDA;
  }
  cudaFree(last_h);
  cudaFree(last_hn);
  last_h = a;
  last_hn = b;
  return B200_OK;
}

b200_status b200_llama::run_layers(b200_kv* kv, int n_req, int T, int n_logits, void* stream) {
  b200_llama* m = this;
  const b200_llama_config& c = cfg;
  const int qd = c.n_heads * c.head_dim, kd = c.n_kv_heads * c.head_dim, qkv_dim = qd + 2 * kd;
  b200_status st;
  cudaStream_t cs = (cudaStream_t)stream;
#define STEP_CAT(cat, call) MODEL_STEP_CAT(cat, call)
#define STEP(call) MODEL_STEP(call)
  STEP(b200_embed_gather(m->embed, m->d_tokens, m->x, T, c.hidden, stream));
  const int fuse_qkv = (m->fuse_qkv_rope && kv->cfg.kv_dtype == B200_KV_BF16 && c.head_dim == 128) ? 1 : 0;
  // The o and down projections also write the RMSNorm their result feeds (fused into their split-K
  // finish pass), so only the first layer normalises x on its own.
  for (int l = 0; l < c.n_layers; ++l) {
    if (l == 0) STEP(b200_rmsnorm(m->x, m->attn_norm[l], m->h, T, c.hidden, c.rms_eps, stream));
    // When the q/k/v projection splits K, its partial sums go straight to RoPE + append (bf16 pools, head_dim 128):
    // same bits, one launch and one pass over the projection's output less.
    b200_qmm_partials parts;
    STEP_CAT(1, b200_qmm_deferred(m->wqkv[l], m->h, T, m->qkv, fuse_qkv, stream, &parts));
    if (parts.pending) {
      STEP_CAT(2, b200_kv_rope_append_partials(kv, l, &parts, m->qkv, qkv_dim, m->d_pos, m->d_row_seq, T, c.n_heads, c.rope_theta, stream));
    } else {
      STEP_CAT(2, b200_kv_rope_append_strided(kv, l, m->qkv, m->qkv + qd, m->qkv + qd + kd, qkv_dim, qkv_dim, qkv_dim, m->d_pos,
                                              m->d_row_seq, T, c.n_heads, c.rope_theta, stream));
    }
    // batches that hold prefill chunks (more rows than requests) take the grouped kernel
    if (T > n_req) { STEP_CAT(0, b200_paged_attn_prefill_strided(kv, l, m->qkv, qkv_dim, m->d_row_seq, m->d_row_ctx, T, m->attn, stream, l > 0)); }
    else { STEP_CAT(0, b200_paged_attn_decode_strided(kv, l, m->qkv, qkv_dim, m->d_row_seq, m->d_row_ctx, T, m->attn, stream, l > 0)); }
    STEP_CAT(1, b200_qmm_residual_norm(m->wo[l], m->attn, T, m->x, m->x, m->ffn_norm[l], c.rms_eps, m->h, stream));
    STEP_CAT(1, b200_qmm(m->wgu[l], m->h, T, m->act, B200_EPI_SWIGLU, nullptr, 0.f, B200_QMM_AUTO, stream));
    if (l + 1 < c.n_layers) {
      STEP_CAT(1, b200_qmm_residual_norm(m->wdown[l], m->act, T, m->x, m->x, m->attn_norm[l + 1], c.rms_eps, m->h, stream));
    } else {
      STEP_CAT(1, b200_qmm(m->wdown[l], m->act, T, m->x, B200_EPI_RESIDUAL, m->x, 0.f, B200_QMM_AUTO, stream));
    }
  }
  STEP(b200_gather_rows(m->x, m->d_logit_row, m->last_h, n_logits, c.hidden, stream));
  STEP(b200_rmsnorm(m->last_h, m->final_norm, m->last_hn, n_logits, c.hidden, c.rms_eps, stream));
  STEP_CAT(1, b200_qmm(m->lm_head, m->last_hn, n_logits, m->logits, B200_EPI_NONE, nullptr, 0.f, B200_QMM_AUTO, stream));
#undef STEP
#undef STEP_CAT
  return B200_OK;
}

extern "C" {

b200_status b200_llama_step(b200_llama* m, b200_kv* kv, const b200_pack_desc* h_desc, int32_t n_req,
                            const uint32_t* h_prefill_tokens, int32_t n_prefill_tokens, uint32_t* h_next_tokens,
                            int32_t* out_free_pages, void* stream) {
  return m->step(kv, h_desc, n_req, h_prefill_tokens, n_prefill_tokens, h_next_tokens, out_free_pages, stream);
}

b200_status b200_llama_forward(b200_llama* m, b200_kv* kv, const b200_pack_desc* d_desc, int32_t n_req, int32_t total_rows,
                               const uint32_t* d_prefill_tokens, void* stream) {
  return m->forward(kv, d_desc, n_req, total_rows, d_prefill_tokens, stream);
}

b200_status b200_llama_set_samplers(b200_llama* m, const b200_sample_params* h_rows, int32_t n_req) { return b200_model_set_samplers(m, h_rows, n_req); }
b200_status b200_llama_last_logprobs(b200_llama* m, float* h_out, int32_t n_req) { return b200_model_last_logprobs(m, h_out, n_req); }

b200_status b200_llama_last_logits(b200_llama* m, void* h_bf16_out, int32_t n_req) {
  if (n_req > m->last_n_req) { b200_set_error("last_logits: %d rows requested, last step had %d", n_req, m->last_n_req); return B200_ERR_CAPACITY; }
  if (n_req > 0) B200_CUDA_TRY(cudaMemcpy(h_bf16_out, m->logits, (size_t)n_req * m->cfg.vocab * 2, cudaMemcpyDeviceToHost));
  return B200_OK;
}

int64_t b200_llama_launch_count(const b200_llama* m) { return m->launches; }
void b200_llama_enable_graphs(b200_llama* m, int32_t on) { m->graphs_on = on != 0; }
void b200_llama_set_fused_qkv_rope(b200_llama* m, int32_t on) {
  m->fuse_qkv_rope = on != 0;
  m->drop_graphs();  // graphs captured with the other setting hold the other kernels
}
void b200_llama_profile_enable(b200_llama* m, int32_t on) { b200_model_profile_enable(m, on); }
b200_status b200_llama_profile_collect(b200_llama* m, double* ms, int64_t* calls) { return b200_model_profile_collect(m, ms, calls); }
void b200_llama_device_buffers(b200_llama* m, b200_pack_desc** d_desc, uint32_t** d_prefill, uint32_t** d_next) {
  b200_model_device_buffers(m, d_desc, d_prefill, d_next);
}

}  // extern "C"
