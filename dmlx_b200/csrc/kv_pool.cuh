// Shared definitions of the device page pool (see kv_pool.cu for the layout).
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <vector>

#include "dmlx_b200.h"

enum { ST_FREE_TOP = 0, ST_ERR = 1, ST_N_TOUCH = 2, ST_N_COW = 3, ST_ATTN_ERR = 4 };

// Shape and place of one layer inside the pool.  A pool made by b200_kv_create has the same shape in every
// layer; one made by b200_kv_create_layers gives each layer its own heads and widths.  `kd` and `vd` are the
// stored widths (elements per token and head), `key_dim` and `value_dim` the model's.
struct KvLayerDev {
  size_t k_off = 0, v_off = 0;  // bytes from the start of k_pool / v_pool
  int heads = 0, kd = 0, vd = 0, key_dim = 0, value_dim = 0;
  int values_in_keys = 0;  // the values are the first value_dim columns of the key rows (vd = 0)
  int rec_elems = 0;       // f32 elements of recurrent state per sequence slot ...
  size_t rec_off = 0;      // ... and where the layer's [max_seqs][rec_elems] start in rec_pool, in elements
};

// Plain-old-data view of the pool, passed to kernels by value.
struct KvDev {
  void* k_pool = nullptr;
  void* v_pool = nullptr;
  float* rec_pool = nullptr;  // recurrent state, [layer][slot][elements]
  float* k_scale = nullptr;
  float* v_scale = nullptr;
  int* free_stack = nullptr;
  int* ref_count = nullptr;
  int* tokens_used = nullptr;
  int* block_table = nullptr;
  int* seq_pages = nullptr;
  int* seq_len = nullptr;
  int* state = nullptr;
  int4* touch_list = nullptr;  // {page, first packed row, rows, first slot in page}
  int2* cow_list = nullptr;    // {source page, private copy}
  const KvLayerDev* layer = nullptr;  // [n_layers]
  int n_layers = 0, n_kv_heads = 0, head_dim = 0, page_size = 0, n_pages = 0, max_seqs = 0, max_pages_per_seq = 0;
  int elem_bytes = 2;
  int max_touch = 0;
};

// Work plan of the attention calls that share a window and a row-group size (attn_window.cu), rebuilt on the
// device once per step: groups of rows, their chunks of pages, and where partial sums go.
struct WindowPlan {
  int window = 0, q_tokens = 1;
  bool fine = false;  // made for the latent kernel
  // group_first [R+2] | chunk_start [R+2] | part_base [R+2] | row_group [R+2] | page_base [R+2] | {n_groups, pages per chunk, pages per
  // worker or 0, -}
  int* buf = nullptr;
};

struct b200_kv {
  uint64_t uid = 0;  // no two pools of a process share it (an address may be used again): captured graphs are kept by it
  b200_kv_config cfg;
  KvDev dev;
  std::vector<KvLayerDev> lay;        // host copy of dev.layer
  std::vector<CUtensorMap> lay_kmap, lay_vmap;  // per-layer 2-D maps (layered bf16 pools): [page*kv_head*32 rows][width]
  std::vector<WindowPlan*> plans;
  bool layered = false;
  uint64_t rec_slot_bytes = 0;        // recurrent state of one slot, all layers
  int max_vd = 0;                     // widest stored value row (sizes the split-K scratch)
  int* d_admin_in = nullptr;
  int* d_admin_out = nullptr;
  int admin_cap = 0;
  // split-K attention scratch
  int* d_chunk_start = nullptr;  // [max_rows + 2]
  float* d_part_o = nullptr;     // [max_chunks][n_q_heads][head_dim]
  float* d_part_ml = nullptr;    // [max_chunks][n_q_heads][2]  (running max in log2 units, sum)
  int max_chunks = 0;
  // row-group plan of the prefill attention path: [3][max_rows + 2] = group_first | part_base | row_group
  int* d_groups = nullptr;
  // 3-D tensor maps over the bf16 pools: [layer][page*kv_head*32 rows][head_dim], box 64 x 32 x 1
  CUtensorMap kmap, vmap;
};

// Internal variants with explicit row strides (elements), used when q/k/v live inside a fused
// projection output.  reuse_plan = 1 skips the split-K planning kernel: the caller guarantees that the
// previous attention call on this pool used the same row arrays (the layers of one model step).
b200_status b200_kv_append_strided(b200_kv* kv, int32_t layer, const void* d_k_rows, const void* d_v_rows,
                                   int32_t k_stride, int32_t v_stride, int32_t total_rows, void* stream);
b200_status b200_kv_rope_append_strided(b200_kv* kv, int32_t layer, void* d_q, const void* d_k_rows, const void* d_v_rows,
                                        int32_t q_stride, int32_t k_stride, int32_t v_stride, const int32_t* d_positions,
                                        const int32_t* d_row_seq, int32_t total_rows, int32_t n_q_heads, float theta, void* stream);
// Attention over one layer of a layered pool (attn_window.cu).  Row r of q ([heads][stored key width] elements, q_stride
// apart) is the token at position row_ctx[r] - 1 of slot row_seq[r]; it sees the last `window` tokens up to itself (0 =
// all), score = (q . k) * scale - slope[head] * distance, and the softmax's denominator also holds exp(sink[head]).
// d_slopes_log2 and d_sinks_log2 (f32 per query head, in units of log2, so multiplied by log2 e) may be null.  The
// output row is [heads][value_dim] in the pool's element type, out_stride elements apart.
struct WindowAttnCall {
  int layer = 0, n_q_heads = 0, window = 0;
  const void* q = nullptr;
  int q_stride = 0;
  float scale = 1.f;
  const float* slopes_log2 = nullptr;
  const float* sinks_log2 = nullptr;
  const float* dist_log2 = nullptr;  // [n_q_heads][dist_len], bias by distance (the last one for all beyond)
  int dist_len = 0;
  void* out = nullptr;
  int out_stride = 0;
  int out_head_stride = 0;  // elements between heads of an output row (0: value_dim)
};
// Builds (once per step) the plan that calls of this window and GQA group size share; `layer` is one of the layers it is
// for (its shape says how many workers the grid has).
b200_status b200_window_attn_plan(b200_kv* kv, int32_t layer, int32_t window, int32_t gqa_group, const int32_t* d_row_seq, const int32_t* d_row_ctx,
                                  int32_t total_rows, void* stream);
// mma = false forces the CUDA-core kernel (which needs no plan).
b200_status b200_window_attn_run(b200_kv* kv, const WindowAttnCall& c, const int32_t* d_row_seq, const int32_t* d_row_ctx, int32_t total_rows,
                                 bool mma, void* stream);
// Whether a layer's pages can go through the tensor-core kernel (bf16, widths up to 256).
bool b200_window_attn_takes_mma(const b200_kv* kv, int32_t layer);
b200_status b200_paged_attn_decode_strided(b200_kv* kv, int32_t layer, const void* d_q, int32_t q_stride,
                                           const int32_t* d_row_seq, const int32_t* d_row_ctx, int32_t total_rows,
                                           void* d_out, void* stream, int32_t reuse_plan);
b200_status b200_paged_attn_prefill_strided(b200_kv* kv, int32_t layer, const void* d_q, int32_t q_stride,
                                            const int32_t* d_row_seq, const int32_t* d_row_ctx, int32_t total_rows,
                                            void* d_out, void* stream, int32_t reuse_plan);
