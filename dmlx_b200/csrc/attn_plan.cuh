// Work items of the paged attention kernels (attn_window.cu builds the plan, attn_latent.cu shares it): groups of consecutive
// rows of one sequence, their pages cut into chunks, and where partial results go.
#pragma once
#include <cuda_bf16.h>

#include "kv_pool.cuh"

constexpr float kAttnLog2e = 1.4426950408889634f;
constexpr float kAttnNone = -1e30f;  // running maximum before any key

struct WinArgs {
  KvDev d;
  KvLayerDev L;
  const __nv_bfloat16* q;
  int q_stride;
  const int* row_seq;
  const int* row_ctx;
  int total_rows, n_q_heads, window;
  int G, head_block, n_blocks;  // query heads per kv head; heads of one MMA tile; tiles per kv head
  const int *group_first, *chunk_start, *part_base, *row_group, *page_base, *hdr;
  float* part_o;   // [slot][q head][L.vd]
  float* part_ml;  // [slot][q head][2]
  float scale_log2;
  const float *slopes, *sinks;
  const float* dist = nullptr;  // [q head][dist_len]: bias by distance, times log2(e); the last one for everything further away
  int dist_len = 0;
  __nv_bfloat16* out;
  int out_stride, out_head;  // elements between rows, between heads of a row
  int stages;                // ring slots: pages per warp, or tiles per CTA
};

__device__ __forceinline__ int first_key(int ctx, int window) { return window > 0 ? max(0, ctx - window) : 0; }

struct WinItem {
  int head, block, seq, first_row, n_rows, ctx0, page_begin, page_end, slot0;  // slot0 < 0: the group has one chunk
};

__device__ __forceinline__ WinItem decode_item(const WinArgs& a, int item, int n_groups) {
  WinItem it;
  const int per_chunk = a.L.heads * a.n_blocks;
  const int chunk = item / per_chunk, rest = item - chunk * per_chunk;
  it.head = rest / a.n_blocks;
  it.block = rest - it.head * a.n_blocks;
  int lo = 0, hi = n_groups - 1;  // last group with chunk_start[group] <= chunk
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (a.chunk_start[mid] <= chunk) lo = mid; else hi = mid - 1;
  }
  it.first_row = a.group_first[lo];
  it.n_rows = a.group_first[lo + 1] - it.first_row;
  it.seq = a.row_seq[it.first_row];
  it.ctx0 = a.row_ctx[it.first_row];
  const int c = chunk - a.chunk_start[lo], n_chunks = a.chunk_start[lo + 1] - a.chunk_start[lo];
  const int p0 = first_key(it.ctx0, a.window) / a.d.page_size;
  const int pages = (it.ctx0 + it.n_rows - 2) / a.d.page_size + 1 - p0;
  const int per_worker = a.hdr[2];
  if (per_worker > 0) {  // the groups' pages lie in one line, cut at multiples of a worker's share
    const int base = a.page_base[lo], k = base / per_worker + c;
    it.page_begin = p0 + max(base, k * per_worker) - base;
    it.page_end = p0 + min(base + pages, (k + 1) * per_worker) - base;
  } else {
    const int each = pages / n_chunks, more = pages - each * n_chunks;  // the first `more` chunks hold one page more
    it.page_begin = p0 + c * each + min(c, more);
    it.page_end = it.page_begin + each + (c < more ? 1 : 0);
  }
  it.slot0 = a.part_base[lo] < 0 ? -1 : a.part_base[lo] + c * it.n_rows;
  return it;
}

// Work items of one worker of a grid whose workers are its blocks: first, behind the last, step.
__device__ __forceinline__ int3 worker_items(const WinArgs& a, int n_groups) {
  const int n_chunks = a.chunk_start[n_groups], per_worker = a.hdr[2];
  if (per_worker == 0) return make_int3(blockIdx.x, n_chunks * a.L.heads * a.n_blocks, gridDim.x);
  auto at = [&](int k) {  // the chunk that starts with worker k's first page
    const int page = k * per_worker;
    int lo = 0, hi = n_groups - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (a.page_base[mid] <= page) lo = mid; else hi = mid - 1;
    }
    return min(n_chunks, a.chunk_start[lo] + k - a.page_base[lo] / per_worker);
  };
  return make_int3(at(blockIdx.x), at(blockIdx.x + 1), 1);
}

// Builds the plan of a (window, tokens per group): items_per_chunk work items per chunk, walked by n_workers.  item_cost and slot_cost:
// what the start and end of a work item, and a row of partial results, cost in pages of one worker's stream.  fine_lengths: for
// kernels that walk worker_items; the plan may then also give every worker an equal share of the pages.
b200_status b200_attn_make_plan(b200_kv* kv, int32_t window, int32_t q_tokens, int32_t items_per_chunk, int32_t n_workers, const int32_t* d_row_seq,
                                const int32_t* d_row_ctx, int32_t total_rows, void* stream, float item_cost, float slot_cost, bool fine_lengths);
// Points the arguments at that plan; false when there is none.
bool b200_attn_use_plan(b200_kv* kv, int32_t window, int32_t q_tokens, bool fine, WinArgs* a);
// Sums the partial results of the groups that were cut.
b200_status b200_attn_combine(b200_kv* kv, const WinArgs& a, void* stream);
