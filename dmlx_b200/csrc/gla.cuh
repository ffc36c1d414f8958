// Gated linear attention and matrix memory over the recurrent state of a layered pool (gla.cu).
#pragma once
#include "kv_pool.cuh"
#include "rows.cuh"

// One layer over the rows of a step.  `src` holds the projection of every row: columns [q | k | v | g | a1] of widths
// heads * dk, heads * dk, heads * dv, heads * dv, rank.  Per head and key channel alpha = sigmoid(W_a2 a1 + b)^(1 / tau);
// S <- diag(alpha) S + k v^T, o = S^T (q * q_scale); the output row is rms_norm(o) * norm * silu(g), [heads][dv].
struct GlaCall {
  int layer = 0, heads = 0, dk = 0, dv = 0, rank = 0;
  MatSrc src;
  const float *a2 = nullptr, *a2_bias = nullptr;  // [heads * dk][rank], [heads * dk]
  const float* norm = nullptr;                    // [dv]
  float q_scale = 1.f, inv_tau = 1.f, eps = 0.f;
  void* out = nullptr;
  int out_stride = 0;
  // Matrix memory: decay and input weight are one number per head and token, made by b200_memory_gates; the keys are summed up
  // beside the state as its column `dv` (their values are ones), and the output is divided by max(|that sum . q|, e^-m) + den_eps,
  // normed, times norm (of every head), sigmoid(g) and out_scale.  src columns from col0: [q | k | v | g].
  const float4* gates = nullptr;  // [rows][heads]
  int col0 = 0;
  float den_eps = 0.f, out_scale = 1.f;
};
// Elements of a matrix memory in a slot's state: S with the key sum ([heads][dk][b200_memory_width(dv)]), then m per head.
constexpr int b200_memory_width(int dv) { return (dv + 1 + 3) / 4 * 4; }
constexpr int b200_memory_elems(int heads, int dk, int dv) { return heads * (dk * b200_memory_width(dv) + 1); }

// Gates of a matrix memory.  src columns [i | f], one per head and kind; log input gate i = cap tanh((z_i + b_i) / cap), log forget
// gate f = log sigmoid(cap tanh((z_f + b_f) / cap)); m_t = max(f + m_(t-1), i) from m = 0, kept in the slot's state.  Written per row
// and head: {f + m_(t-1) - m_t, e^(i - m_t), e^(-m_t), -}.
struct MemoryGates {
  int layer = 0, heads = 0, m_off = 0;  // m_off: where m starts in the slot's state
  MatSrc src;
  const float* bias = nullptr;  // [2 heads]
  float cap = 1.f;
  float4* out = nullptr;
};
b200_status b200_memory_gates(b200_kv* kv, const MemoryGates& g, const int32_t* d_cu, const int32_t* d_row_seq, const int32_t* d_pos, int n_req,
                              int total_rows, void* stream);

// Buffers of the chunk-wise path, shared by the layers of a model: made for a number of rows and requests.
struct GlaScratch {
  int max_rows = 0, max_reqs = 0, max_chunks = 0;
  size_t chunk_bytes = 0, v_bytes = 0, o_elems = 0;  // per (chunk, head); per row
  unsigned char *chunks = nullptr, *values = nullptr;
  float* o = nullptr;
  int4* plan = nullptr;      // [max_chunks] {first row, rows, request, -}
  int* first_chunk = nullptr;  // [max_reqs + 1]
  // delta rule (delta.cuh): q, k and v of a row behind their convolutions, and {log decay, beta} per head
  size_t row_elems = 0;
  int gate_heads = 0;
  float* rows = nullptr;
  float2* gates = nullptr;
  bool alloc();              // false: out of memory
  void need(int heads, int dk, int dv, bool delta = false);  // before alloc: a layer of this shape will use it
  void need_delta(int heads, int kv_heads, int dk, int dv, bool chunks);
  void free();
};

// A step's rows are cut once for all layers.  Portions of more than `step_tokens` tokens go chunk by chunk on the tensor
// cores (bf16), shorter ones token by token.
b200_status b200_gla_plan(GlaScratch& g, const int32_t* d_cu, int n_req, int total_rows, void* stream);
b200_status b200_gla_run(b200_kv* kv, const GlaScratch& g, const GlaCall& c, const int32_t* d_cu, const int32_t* d_row_seq,
                         const int32_t* d_pos, int n_req, int total_rows, bool chunked, void* stream);
// Whether a layer's shape fits the chunk-wise kernels.
bool b200_gla_takes_chunks(int dk, int dv, int elem_bytes);
constexpr int kGlaStepTokens = 4;
