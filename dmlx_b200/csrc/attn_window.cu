// Paged attention for layers with a sliding window, a distance bias (linear, or by a table) and a learned sink, keys and values of different
// widths, and any GQA group; decode rows and prefill chunks through one path.
//
// Rows are grouped: consecutive rows of one sequence (a prefill chunk) share a pass over the pages, a decoded token is a
// group of its own.  The 16 rows of an MMA tile carry (token of the group) x (query head of the kv head's GQA group), so
// a group holds floor(16 / G) tokens; groups with more than 16 query heads per kv head are cut into head blocks of 16.
// A group's key range is [first row's window start, last row's position]; it is cut into chunks of pages, and a work item
// is (chunk, kv head, head block), walked by a persistent grid whose warps are independent workers (each with its own
// ring of TMA-staged pages, as in paged_attn.cu).  A group of one chunk is normalised and written by the kernel itself; the
// partial (max, sum, out) of longer ones go through scratch to a combine pass.  The sink joins the denominator exactly
// once, where a row is normalised.
//
// Scores, biases and softmax are f32.  The weights enter the P V product as two bf16 terms (the rounded weight and what
// the rounding left over), so they carry 16 bits of mantissa instead of 8.
//
// attn_simt_kernel does the same on CUDA cores for any width and for f32 pools.
#include <cuda_bf16.h>

#include <algorithm>
#include <cmath>
#include <type_traits>

#include "attn_latent.cuh"
#include "attn_plan.cuh"
#include "common.h"
#include "kv_pool.cuh"
#include "ptx.cuh"
#include "tma.cuh"

namespace {

constexpr float kLog2e = kAttnLog2e, kNone = kAttnNone;

// ---- plan ------------------------------------------------------------------------------------------------
template <bool MAX>
__device__ int scan_incl(int v, int* warp_buf) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int inc = v;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int t = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc = MAX ? max(inc, t) : inc + t;
  }
  if (lane == 31) warp_buf[warp] = inc;
  __syncthreads();
  if (warp == 0) {
    int w = lane < (int)(blockDim.x >> 5) ? warp_buf[lane] : (MAX ? -1 : 0);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int t = __shfl_up_sync(0xffffffffu, w, o);
      if (lane >= o) w = MAX ? max(w, t) : w + t;
    }
    const int ex = __shfl_up_sync(0xffffffffu, w, 1);
    warp_buf[lane] = lane == 0 ? (MAX ? -1 : 0) : ex;
  }
  __syncthreads();
  const int r = MAX ? max(warp_buf[warp], inc) : warp_buf[warp] + inc;
  __syncthreads();
  return r;
}

// Pages of a group's key range.
__device__ __forceinline__ int group_pages(int ctx_first, int ctx_last, int window, int page_size) {
  return (max(ctx_last, 1) - 1) / page_size - first_key(ctx_first, window) / page_size + 1;
}

// Chunk lengths the plan tries: few and coarse where a grid has many workers, fine steps where a work item is a large part of a
// worker's load and the number of waves decides.
struct CoarseLengths {
  static constexpr int kCand = 6;  // 4, 8, 16, 32, 64 pages, uncut
  static __device__ __forceinline__ int at(int k) { return 4 << k; }
};
struct FineLengths {
  static constexpr int kCand = 18;  // 8, 12, 16 .. 64 pages, 80, 96, uncut
  static __device__ __forceinline__ int at(int k) { return k < 15 ? 8 + 4 * k : 80 + 16 * (k - 15); }
};

// Groups of rows and their chunks.  A group's pages are cut evenly into ceil(pages / ppc) chunks.  ppc is the candidate with
// the smallest estimated time, in pages of one worker's stream: the average load or the longest item, half an item for
// the uneven end of the walk, a page and a bit per item for its start and end, and, where groups are cut, the partial sums
// and the combine pass.  It doubles until the partial slots fit the scratch (uncut groups need none), so a step always fits.
template <typename Lengths>
__global__ void __launch_bounds__(1024) window_plan_kernel(const int* __restrict__ row_seq, const int* __restrict__ row_ctx, int total_rows,
                                                           int page_size, int window, int q_tokens, int items_per_chunk,
                                                           int n_workers, int forced_ppc, int max_slots, float item_cost, float slot_cost, int* __restrict__ group_first,
                                                           int* __restrict__ chunk_start, int* __restrict__ part_base,
                                                           int* __restrict__ row_group, int* __restrict__ page_base, int* __restrict__ hdr) {
  __shared__ int warp_buf[32];
  __shared__ int carry_start, carry_groups, carry_chunks, carry_slots, carry_pages, s_share;
  const int tid = threadIdx.x;
  if (tid == 0) { carry_start = -1; carry_groups = 0; s_share = 0; }
  __syncthreads();
  for (int base = 0; base < total_rows; base += blockDim.x) {
    const int i = base + tid;
    const bool valid = i < total_rows;
    const bool joinable = valid && i > 0 && row_seq[i] == row_seq[i - 1] && row_ctx[i] == row_ctx[i - 1] + 1;
    const int run_start = max(scan_incl<true>(valid && !joinable ? i : -1, warp_buf), carry_start);
    const int head = valid && ((i - run_start) % q_tokens == 0) ? 1 : 0;
    const int heads_incl = scan_incl<false>(head, warp_buf);
    const int gid = carry_groups + heads_incl - 1;
    if (valid) {
      row_group[i] = gid;
      if (head) group_first[gid] = i;
    }
    __syncthreads();
    if (tid == blockDim.x - 1) { carry_start = run_start; carry_groups += heads_incl; }
    __syncthreads();
  }
  const int n_groups = carry_groups;
  if (tid == 0) group_first[n_groups] = total_rows;
  __syncthreads();
  int ppc = 0x3fffffff;
  if (forced_ppc > 0) {
    ppc = forced_ppc;
  } else {
    constexpr int kCand = Lengths::kCand;
    long long chunks[kCand] = {}, slots[kCand] = {}, pages_sum = 0;
    int longest = 0;
    for (int g = tid; g < n_groups; g += blockDim.x) {
      const int first = group_first[g], next = group_first[g + 1];
      const int pages = group_pages(row_ctx[first], row_ctx[next - 1], window, page_size);
      pages_sum += pages;
      longest = max(longest, pages);
#pragma unroll
      for (int k = 0; k < kCand; ++k) {
        const int c = k == kCand - 1 ? 1 : (pages + Lengths::at(k) - 1) / Lengths::at(k);
        chunks[k] += c;
        slots[k] += c > 1 ? c * (next - first) : 0;
      }
    }
    __shared__ long long s_red[32][2 * kCand + 2];
#pragma unroll
    for (int k = 0; k < 2 * kCand + 2; ++k) {
      long long v = k < kCand ? chunks[k < kCand ? k : 0] : (k < 2 * kCand ? slots[k < 2 * kCand ? (k >= kCand ? k - kCand : 0) : 0] : (k == 2 * kCand ? pages_sum : longest));
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const long long w = __shfl_xor_sync(0xffffffffu, v, o);
        v = k == 2 * kCand + 1 ? (v > w ? v : w) : v + w;
      }
      if ((tid & 31) == 0) s_red[tid >> 5][k] = v;
    }
    __syncthreads();
    if (tid < 2 * kCand + 2) {
      long long sum = 0, most = 0;
      for (int w = 0; w < (int)(blockDim.x >> 5); ++w) {
        const long long v = s_red[w][tid];
        sum += v;
        most = most > v ? most : v;
      }
      s_red[0][tid] = tid == 2 * kCand + 1 ? most : sum;
    }
    __syncthreads();
    if (tid == 0) {
      const long long* tot = s_red[0];
      const float per = (float)items_per_chunk / (float)n_workers, load = (float)tot[2 * kCand] * per;
      float best = 3.4e38f;
      for (int k = 0; k < kCand; ++k) {
        const float length = fminf(k == kCand - 1 ? 1e9f : (float)Lengths::at(k), (float)tot[2 * kCand + 1]);
        const float items = (float)tot[k] * per;
        float t;
        if (kCand > 6) {  // whole waves of average items, the longest last
          const float waves = ceilf(items), mean = (float)tot[2 * kCand] / (float)tot[k];
          t = (waves - 1.f) * mean + length + item_cost * waves;
        } else {
          t = fmaxf(load, length) + (items > 1.f ? 0.5f * length : 0.f) + item_cost * items;
        }
        if (tot[kCand + k] > 0) t += 3.f + slot_cost * (float)tot[kCand + k] * per;
        if (t < best) { best = t; carry_chunks = k; }
      }
      // Equal shares: about one more item per worker than whole groups would make.  (Not for prompts: there the workers should walk
      // neighbouring groups side by side, which read the same pages.)
      if (kCand > 6 && items_per_chunk == 1 && n_groups <= 4 * n_workers) {
        const long long pages = tot[2 * kCand];
        const int share = max((int)((pages + n_workers - 1) / n_workers), 4);
        const float cuts = (float)pages / (float)share, items = ((float)n_groups + cuts) / (float)n_workers;
        const float rows_cut = fminf(2.f * cuts, (float)n_groups + cuts) * (float)total_rows / (float)n_groups;
        if ((float)share + item_cost * fmaxf(items, 1.f) + 3.f + slot_cost * rows_cut / (float)n_workers < best) s_share = share;
      }
    }
    __syncthreads();
    ppc = carry_chunks == kCand - 1 ? 0x3fffffff : Lengths::at(carry_chunks);
    __syncthreads();
  }
  int share = s_share;
  for (int round = 0; round < 32; ++round) {
    if (tid == 0) { carry_chunks = 0; carry_slots = 0; carry_pages = 0; }
    __syncthreads();
    for (int base = 0; base < n_groups; base += blockDim.x) {
      const int g = base + tid;
      int chunks = 0, slots = 0, pages = 0, rows = 0;
      if (g < n_groups) {
        const int first = group_first[g], next = group_first[g + 1];
        pages = group_pages(row_ctx[first], row_ctx[next - 1], window, page_size);
        rows = next - first;
      }
      if (share > 0) {
        const int base_page = carry_pages + scan_incl<false>(pages, warp_buf) - pages;
        if (g < n_groups) {
          page_base[g] = base_page;
          chunks = (base_page + pages - 1) / share - base_page / share + 1;
        }
      } else {
        chunks = pages / ppc + (pages % ppc ? 1 : 0);
      }
      slots = chunks > 1 ? chunks * rows : 0;
      const int c_incl = scan_incl<false>(chunks, warp_buf);
      const int s_incl = scan_incl<false>(slots, warp_buf);
      if (g < n_groups) {
        chunk_start[g] = carry_chunks + c_incl - chunks;
        part_base[g] = slots > 0 ? carry_slots + s_incl - slots : -1;
      }
      __syncthreads();
      if (tid == blockDim.x - 1) { carry_chunks += c_incl; carry_slots += s_incl; }
      const int page_sum = scan_incl<false>(pages, warp_buf);
      if (tid == blockDim.x - 1) carry_pages += page_sum;
      __syncthreads();
    }
    if (carry_slots <= max_slots) break;
    __syncthreads();
    ppc = ppc > (1 << 28) ? ppc : ppc * 2;
    share = share > (1 << 28) ? share : share * 2;
  }
  if (tid == 0) {
    chunk_start[n_groups] = carry_chunks;
    hdr[0] = n_groups;
    hdr[1] = ppc;
    hdr[2] = share;
  }
}

// ---- tensor-core kernel ------------------------------------------------------------------------------------
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// (p0, p1) as two bf16 pairs: the rounded values and the remainders.
__device__ __forceinline__ void split_bf16(float p0, float p1, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(p0 - f.x, p1 - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

// KB, VB: 64-column boxes a key / value row may take (1, 2 or 4); the steps beyond the layer's own widths are skipped.
// A block is as many independent warps as its shared memory and registers feed.  TABLE: the layer has a bias by distance.
constexpr int most_warps(int kb, int vb) { return kb + vb == 2 ? 12 : (kb + vb == 3 ? 9 : 8); }
template <int KB, int VB, bool TABLE>
__global__ void __launch_bounds__(most_warps(KB, VB) * 32, 1)
    window_attn_mma_kernel(const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap, WinArgs a) {
  constexpr int KS = KB * 4;  // 16-column steps of Q K^T
  constexpr int NO = VB * 8;  // 8-column tiles of the output
  const int n_kb = (a.L.kd + 63) / 64, n_vb = (a.L.vd + 63) / 64, n_ks = a.L.kd / 16, n_vs = a.L.vd / 16;
  const int warps = blockDim.x >> 5, kStages = a.stages, k_tile = n_kb * 4096, stage_bytes = (n_kb + n_vb) * 4096;

  extern __shared__ unsigned char smem_dyn[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_dyn) + 1023) & ~(uintptr_t)1023);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane >> 2, t = lane & 3;
  unsigned char* my_tiles = smem + (size_t)warp * kStages * stage_bytes;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + (size_t)warps * kStages * stage_bytes) + warp * kStages;
  const int H = a.L.heads;
  const int n_groups = a.hdr[0];
  const int n_items = a.chunk_start[n_groups] * H * a.n_blocks;
  const int worker = blockIdx.x * warps + warp, n_workers = gridDim.x * warps;

  if (lane == 0) {
    for (int s = 0; s < kStages; ++s) ptx::mbar_init(&full_bar[s], 1);
    ptx::mbar_fence_init();
  }
  __syncwarp();

  // producer cursor (all lanes track it, lane 0 issues); the lanes hold the page ids of a window of 32 pages of the
  // item's chunk, refilled every 32 pages
  int p_item = worker, p_page = 0, p_end = 0, p_begin = 0, p_head = 0, p_pid = 0, p_seq = 0;
  int prod_s = 0;  // slot of the next page
  auto producer_enter_item = [&]() {
    if (p_item < n_items) {
      const WinItem it = decode_item(a, p_item, n_groups);
      p_begin = it.page_begin; p_page = it.page_begin; p_end = it.page_end; p_head = it.head; p_seq = it.seq;
      const int pg = it.page_begin + lane;
      if (pg < it.page_end) p_pid = a.d.block_table[(size_t)it.seq * a.d.max_pages_per_seq + pg];
    }
  };
  auto produce_one = [&]() {
    if (p_item >= n_items) return;
    const int rel = p_page - p_begin;
    if (rel > 0 && (rel & 31) == 0) {
      const int pg = p_page + lane;
      if (pg < p_end) p_pid = a.d.block_table[(size_t)p_seq * a.d.max_pages_per_seq + pg];
    }
    const int pid = __shfl_sync(0xffffffffu, p_pid, rel & 31);
    const int s = prod_s;
    if (lane == 0) {
      ptx::fence_proxy_async_smem();
      unsigned char* kd = my_tiles + (size_t)s * stage_bytes;
      const int row0 = (pid * H + p_head) * 32;
      ptx::mbar_expect_tx(&full_bar[s], stage_bytes);
      for (int b = 0; b < n_kb; ++b) ptx::tma_load_2d(kd + b * 4096, &kmap, b * 64, row0, &full_bar[s]);
      for (int b = 0; b < n_vb; ++b) ptx::tma_load_2d(kd + k_tile + b * 4096, &vmap, b * 64, row0, &full_bar[s]);
    }
    if (++prod_s == kStages) prod_s = 0;
    p_page += 1;
    if (p_page >= p_end) {
      p_item += n_workers;
      producer_enter_item();
    }
  };
  producer_enter_item();
  for (int i = 0; i < kStages; ++i) produce_one();

  bool alive = true;
  int cons_s = 0;
  uint32_t cons_ph = 0;
  const int ld_r = lane & 7, ld_m = lane >> 3;
  // MMA rows g and g+8 of this lane: (token of the group, query head within the block)
  const int hb = a.head_block;
  const int tokA = g / hb, headA = g - tokA * hb, tokB = (g + 8) / hb, headB = (g + 8) - tokB * hb;
  for (int item = worker; item < n_items && alive; item += n_workers) {
    const WinItem it = decode_item(a, item, n_groups);
    const int h0 = it.head * a.G + it.block * hb;  // first query head of the block
    const int heads_here = min(hb, a.G - it.block * hb);
    const bool onA = tokA < it.n_rows && headA < heads_here, onB = tokB < it.n_rows && headB < heads_here;
    const int ctxA = onA ? it.ctx0 + tokA : 0, ctxB = onB ? it.ctx0 + tokB : 0;
    const int loA = first_key(ctxA, a.window), loB = first_key(ctxB, a.window);
    const int qhA = h0 + (onA ? headA : 0), qhB = h0 + (onB ? headB : 0);
    const int lo_last = first_key(it.ctx0 + it.n_rows - 1, a.window);  // the latest window start of the group
    const bool any_b = it.n_rows * hb > 8;                            // rows 8..15 of the tile carry something
    const float slA = a.slopes ? a.slopes[qhA] : 0.f, slB = a.slopes ? a.slopes[qhB] : 0.f;
    // the first key that some row of the group sees at a distance of its own
    const int near_from = TABLE ? it.ctx0 - (a.dist_len - 1) : 0;
    uint32_t qa0[KS], qa1[KS], qa2[KS], qa3[KS];
    {
      const uint32_t* qA = reinterpret_cast<const uint32_t*>(a.q + (size_t)(it.first_row + (onA ? tokA : 0)) * a.q_stride + (size_t)qhA * a.L.kd);
      const uint32_t* qB = reinterpret_cast<const uint32_t*>(a.q + (size_t)(it.first_row + (onB ? tokB : 0)) * a.q_stride + (size_t)qhB * a.L.kd);
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        const bool in = ks < n_ks;
        qa0[ks] = onA && in ? qA[ks * 8 + t] : 0u;
        qa2[ks] = onA && in ? qA[ks * 8 + 4 + t] : 0u;
        qa1[ks] = onB && in ? qB[ks * 8 + t] : 0u;
        qa3[ks] = onB && in ? qB[ks * 8 + 4 + t] : 0u;
      }
    }
    float o[NO][4];
#pragma unroll
    for (int j = 0; j < NO; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
    float mA = kNone, lA = 0.f, mB = kNone, lB = 0.f;

    for (int pg = it.page_begin; pg < it.page_end; ++pg) {
      const int s = cons_s;
      alive = ptx::mbar_wait(&full_bar[s], cons_ph);
      if (!alive) break;
      const uint32_t kbase = ptx::smem_u32(my_tiles + (size_t)s * stage_bytes), vbase = kbase + k_tile;
      float sc[4][4];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) { sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f; }
#pragma unroll
      for (int kk = 0; kk < KS / 2; ++kk) {
        if (2 * kk < n_ks) {
#pragma unroll
          for (int nt = 0; nt < 4; ++nt) {
            const int row = nt * 8 + ld_r, cc = 4 * kk + ld_m;
            uint32_t b[4];
            ldsm4(kbase + (cc >> 3) * 4096 + row * 128 + (((cc & 7) ^ (row & 7)) << 4), b);
            mma16816(sc[nt], qa0[2 * kk], qa1[2 * kk], qa2[2 * kk], qa3[2 * kk], b[0], b[1]);
            mma16816(sc[nt], qa0[2 * kk + 1], qa1[2 * kk + 1], qa2[2 * kk + 1], qa3[2 * kk + 1], b[2], b[3]);
          }
        }
      }
      // ---- online softmax on rows g (A) and, where the tile has any, g+8 (B), each with its own window and bias ----
      const int tok0 = pg * 32;
      uint32_t ph[2][4], pl[2][4];
      // a page every row of the group sees whole needs no masks; beyond the reach of a distance table all keys have the same bias
      const int kind = TABLE && tok0 + 31 >= near_from ? 2 : (tok0 + 32 > it.ctx0 || tok0 < lo_last ? 1 : 0);
      auto row_softmax = [&](auto kind_tag, auto half_tag, float& m, float& l, int ctx, int lo, float slope, int qh) -> float {
        constexpr bool EDGE = decltype(kind_tag)::value > 0, NEAR = decltype(kind_tag)::value == 2;
        constexpr int E0 = decltype(half_tag)::value;  // 0: row g, 1: row g + 8
        float mx = kNone;
        const float* tab = TABLE ? a.dist + (size_t)qh * a.dist_len : nullptr;
        float b0 = slope * (float)(tok0 + 2 * t - (ctx - 1));  // exact integers; the bias of the lane's first key
        if constexpr (TABLE && !NEAR) b0 += tab[a.dist_len - 1];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int tok = tok0 + nt * 8 + 2 * t + e;
            float v;
            if constexpr (NEAR) v = fmaf(sc[nt][2 * E0 + e], a.scale_log2, tab[min(max(ctx - 1 - tok, 0), a.dist_len - 1)]);
            else v = sc[nt][2 * E0 + e] * a.scale_log2 + fmaf(slope, (float)(nt * 8 + e), b0);
            if (EDGE) v = tok < ctx && tok >= lo ? v : kNone;
            sc[nt][2 * E0 + e] = v;
            mx = fmaxf(mx, v);
          }
        }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m, mx), corr = ex2(m - m_new);
        float ps = 0.f;
#pragma unroll
        for (int kt = 0; kt < 2; ++kt) {
          float p[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float v = sc[2 * kt + (e >> 1)][2 * E0 + (e & 1)];
            p[e] = ex2(v - m_new);
            if (EDGE) p[e] = v > kNone ? p[e] : 0.f;
            ps += p[e];
          }
          split_bf16(p[0], p[1], ph[kt][E0], pl[kt][E0]);
          split_bf16(p[2], p[3], ph[kt][2 + E0], pl[kt][2 + E0]);
        }
        l = l * corr + ps;
        m = m_new;
        return corr;
      };
      using T0 = std::integral_constant<int, 0>;
      using T1 = std::integral_constant<int, 1>;
      using T2 = std::integral_constant<int, 2>;
      auto softmax = [&](auto half_tag, float& m, float& l, int ctx, int lo, float slope, int qh) -> float {
        if constexpr (TABLE) {
          if (kind == 2) return row_softmax(T2{}, half_tag, m, l, ctx, lo, slope, qh);
        }
        return kind == 0 ? row_softmax(T0{}, half_tag, m, l, ctx, lo, slope, qh) : row_softmax(T1{}, half_tag, m, l, ctx, lo, slope, qh);
      };
      const float corrA = softmax(T0{}, mA, lA, ctxA, loA, slA, qhA);
      float corrB = 1.f;
      if (any_b) {
        corrB = softmax(T1{}, mB, lB, ctxB, loB, slB, qhB);
      } else {
#pragma unroll
        for (int kt = 0; kt < 2; ++kt) { ph[kt][1] = ph[kt][3] = pl[kt][1] = pl[kt][3] = 0u; }
      }
      if (__any_sync(0xffffffffu, corrA != 1.f || corrB != 1.f)) {
#pragma unroll
        for (int j = 0; j < NO; ++j) { o[j][0] *= corrA; o[j][1] *= corrA; o[j][2] *= corrB; o[j][3] *= corrB; }
      }
#pragma unroll
      for (int jj = 0; jj < NO / 2; ++jj) {
        if (jj < n_vs) {
#pragma unroll
          for (int kt = 0; kt < 2; ++kt) {
            const int row = kt * 16 + (ld_m & 1) * 8 + ld_r, cc = 2 * jj + (ld_m >> 1);
            uint32_t b[4];
            ldsm4_trans(vbase + (cc >> 3) * 4096 + row * 128 + (((cc & 7) ^ (row & 7)) << 4), b);
            mma16816(o[2 * jj], ph[kt][0], ph[kt][1], ph[kt][2], ph[kt][3], b[0], b[1]);
            mma16816(o[2 * jj + 1], ph[kt][0], ph[kt][1], ph[kt][2], ph[kt][3], b[2], b[3]);
            mma16816(o[2 * jj], pl[kt][0], pl[kt][1], pl[kt][2], pl[kt][3], b[0], b[1]);
            mma16816(o[2 * jj + 1], pl[kt][0], pl[kt][1], pl[kt][2], pl[kt][3], b[2], b[3]);
          }
        }
      }
      __syncwarp();
      if (++cons_s == kStages) { cons_s = 0; cons_ph ^= 1u; }
      produce_one();  // refill the slot just drained
    }
    if (!alive) break;
    lA += __shfl_xor_sync(0xffffffffu, lA, 1);
    lA += __shfl_xor_sync(0xffffffffu, lA, 2);
    lB += __shfl_xor_sync(0xffffffffu, lB, 1);
    lB += __shfl_xor_sync(0xffffffffu, lB, 2);
    auto store = [&](bool on, int tok, int qh, float m, float l, int e0) {
      if (!on) return;
      if (it.slot0 < 0) {
        float f = 1.f;
        if (a.sinks) {
          const float sk = a.sinks[qh], mm = fmaxf(m, sk);
          f = exp2f(m - mm);
          l = l * f + exp2f(sk - mm);
        }
        const float inv = l > 0.f ? f / l : 0.f;
        __nv_bfloat16* dst = a.out + (size_t)(it.first_row + tok) * a.out_stride + (size_t)qh * a.out_head;
#pragma unroll
        for (int j = 0; j < NO; ++j) {
          const int c = j * 8 + 2 * t;
          if ((a.L.value_dim & 1) == 0) {
            if (c < a.L.value_dim) *reinterpret_cast<__nv_bfloat162*>(dst + c) = __floats2bfloat162_rn(o[j][e0] * inv, o[j][e0 + 1] * inv);
          } else {
            if (c < a.L.value_dim) dst[c] = __float2bfloat16(o[j][e0] * inv);
            if (c + 1 < a.L.value_dim) dst[c + 1] = __float2bfloat16(o[j][e0 + 1] * inv);
          }
        }
      } else {
        const size_t pidx = (size_t)(it.slot0 + tok) * a.n_q_heads + qh;
#pragma unroll
        for (int j = 0; j < NO; ++j)
          if (j * 8 < a.L.vd) *reinterpret_cast<float2*>(a.part_o + pidx * a.L.vd + j * 8 + 2 * t) = make_float2(o[j][e0], o[j][e0 + 1]);
        if (t == 0) { a.part_ml[pidx * 2] = m; a.part_ml[pidx * 2 + 1] = l; }
      }
    };
    store(onA, tokA, qhA, mA, lA, 0);
    store(onB, tokB, qhB, mB, lB, 2);
  }
  if (!alive && lane == 0) atomicExch(a.d.state + ST_ATTN_ERR, B200_ERR_DEVICE_FLAGGED);
}

// One warp per (row, query head) of the groups that were cut into several chunks.
__global__ void __launch_bounds__(256) window_combine_kernel(WinArgs a) {
  const int lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (w >= (long long)a.total_rows * a.n_q_heads || a.d.state[ST_ATTN_ERR] != 0) return;
  const int row = (int)(w / a.n_q_heads), qh = (int)(w - (long long)row * a.n_q_heads);
  const int grp = a.row_group[row];
  if (a.part_base[grp] < 0) return;
  const int first = a.group_first[grp], size = a.group_first[grp + 1] - first, n_chunks = a.chunk_start[grp + 1] - a.chunk_start[grp];
  const size_t slot0 = (size_t)a.part_base[grp] + (row - first);
  float mm = a.sinks ? a.sinks[qh] : kNone;
  for (int c = lane; c < n_chunks; c += 32) mm = fmaxf(mm, a.part_ml[((slot0 + (size_t)c * size) * a.n_q_heads + qh) * 2]);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffffu, mm, o));
  float l = 0.f;
  for (int c = lane; c < n_chunks; c += 32) {
    const size_t pidx = (slot0 + (size_t)c * size) * a.n_q_heads + qh;
    l += a.part_ml[pidx * 2 + 1] * exp2f(a.part_ml[pidx * 2] - mm);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
  if (a.sinks) l += exp2f(a.sinks[qh] - mm);
  const float inv = l > 0.f ? 1.0f / l : 0.f;
  __nv_bfloat16* dst = a.out + (size_t)row * a.out_stride + (size_t)qh * a.out_head;
  for (int v0 = blockIdx.y * 128; v0 < a.L.vd; v0 += gridDim.y * 128) {  // four columns per lane
    const int v = v0 + 4 * lane;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (v < a.L.vd) {
#pragma unroll 4
      for (int c = 0; c < n_chunks; ++c) {
        const size_t pidx = (slot0 + (size_t)c * size) * a.n_q_heads + qh;
        const float wgt = exp2f(a.part_ml[pidx * 2] - mm);
        const float4 p = *reinterpret_cast<const float4*>(a.part_o + pidx * a.L.vd + v);
        acc[0] += p.x * wgt; acc[1] += p.y * wgt; acc[2] += p.z * wgt; acc[3] += p.w * wgt;
      }
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (v + e < a.L.value_dim) dst[v + e] = __float2bfloat16(acc[e] * inv);
    }
  }
}

// ---- CUDA-core kernel: any width, bf16 or f32 pools -----------------------------------------------------------
__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(__nv_bfloat16 x) { return __bfloat162float(x); }
__device__ __forceinline__ void put(float* p, float x) { *p = x; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float x) { *p = __float2bfloat16(x); }

struct SimtArgs {
  KvDev d;
  KvLayerDev L;
  const void* q;
  int q_stride;
  const int* row_seq;
  const int* row_ctx;
  int total_rows, n_q_heads, window;
  float scale;
  const float *slopes_log2, *sinks_log2, *dist_log2;
  int dist_len;
  void* out;
  int out_stride, out_head_stride;
};

// One warp per (row, query head): 32 keys at a time (one per lane) for the scores, value columns over the lanes for the
// weighted sum; query and output row in shared memory.
template <typename T>
__global__ void __launch_bounds__(128) attn_simt_kernel(SimtArgs a) {
  extern __shared__ float sh[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, kd = a.L.key_dim, vd = a.L.value_dim;
  float* q = sh + warp * (kd + vd);
  float* o = q + kd;
  const long long w = (long long)blockIdx.x * 4 + warp;
  if (w >= (long long)a.total_rows * a.n_q_heads) return;
  const int row = (int)(w / a.n_q_heads), qh = (int)(w - (long long)row * a.n_q_heads), head = qh / (a.n_q_heads / a.L.heads);
  const T* qg = (const T*)a.q + (size_t)row * a.q_stride + (size_t)qh * a.L.kd;
  for (int c = lane; c < kd; c += 32) q[c] = to_f(qg[c]);
  for (int c = lane; c < vd; c += 32) o[c] = 0.f;
  __syncwarp();
  const int seq = a.row_seq[row], ctx = a.row_ctx[row], lo = first_key(ctx, a.window);
  if (seq < 0 || seq >= a.d.max_seqs || (ctx + 31) / 32 > a.d.seq_pages[seq]) return;  // reservation failed: the step is flagged
  const int* table = a.d.block_table + (size_t)seq * a.d.max_pages_per_seq;
  const T* kp = (const T*)((const char*)a.d.k_pool + a.L.k_off);
  const T* vp = a.L.values_in_keys ? kp : (const T*)((const char*)a.d.v_pool + a.L.v_off);
  const int v_row = a.L.values_in_keys ? a.L.kd : a.L.vd;
  const float slope = a.slopes_log2 ? a.slopes_log2[qh] : 0.f, scale = a.scale * kLog2e;
  const float* tab = a.dist_log2 ? a.dist_log2 + (size_t)qh * a.dist_len : nullptr;
  float m = kNone, l = 0.f;
  for (int pg = lo / 32; pg * 32 < ctx; ++pg) {
    const int tok = pg * 32 + lane;
    const size_t tile = ((size_t)table[pg] * a.L.heads + head) * 32;
    const bool on = tok >= lo && tok < ctx;
    float s = kNone;
    if (on) {
      const T* kr = kp + (tile + lane) * a.L.kd;
      float acc = 0.f;
      for (int c = 0; c < kd; ++c) acc = fmaf(q[c], to_f(kr[c]), acc);
      s = acc * scale - slope * (float)(ctx - 1 - tok);
      if (tab) s += tab[min(ctx - 1 - tok, a.dist_len - 1)];
    }
    float mx = s;
#pragma unroll
    for (int b = 16; b > 0; b >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, b));
    const float m_new = fmaxf(m, mx), corr = exp2f(m - m_new), p = on ? exp2f(s - m_new) : 0.f;
    float ps = p;
#pragma unroll
    for (int b = 16; b > 0; b >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, b);
    l = l * corr + ps;
    m = m_new;
    const int k0 = max(lo - pg * 32, 0), k1 = min(ctx - pg * 32, 32);
    for (int c0 = 0; c0 < vd; c0 += 32) {
      const int c = c0 + lane;
      float acc = c < vd ? o[c] * corr : 0.f;
      for (int k = k0; k < k1; ++k) {
        const float pk = __shfl_sync(0xffffffffu, p, k);
        if (c < vd) acc = fmaf(pk, to_f(vp[(tile + k) * v_row + c]), acc);
      }
      if (c < vd) o[c] = acc;
    }
    __syncwarp();
  }
  float f = 1.f;
  if (a.sinks_log2) {
    const float sk = a.sinks_log2[qh], mm = fmaxf(m, sk);
    f = exp2f(m - mm);
    l = l * f + exp2f(sk - mm);
  }
  T* out = (T*)a.out + (size_t)row * a.out_stride + (size_t)qh * a.out_head_stride;
  for (int c = lane; c < vd; c += 32) put(out + c, l > 0.f ? o[c] * f / l : 0.f);
}

int g_sms = 0;
b200_status sm_count() {
  if (g_sms == 0) {
    int dev = 0;
    B200_CUDA_TRY(cudaGetDevice(&dev));
    B200_CUDA_TRY(cudaDeviceGetAttribute(&g_sms, cudaDevAttrMultiProcessorCount, dev));
  }
  return B200_OK;
}

int head_block_of(int gqa) { return std::min(gqa, 16); }
int q_tokens_of(int gqa) { return gqa >= 16 ? 1 : 16 / gqa; }

WindowPlan* find_plan(b200_kv* kv, int window, int q_tokens, bool fine) {
  for (WindowPlan* p : kv->plans)
    if (p->window == window && p->q_tokens == q_tokens && p->fine == fine) return p;
  return nullptr;
}

// Warps of a block and ring slots per warp, by the 4 KiB boxes of a staged page (keys + values).  The warps are
// bound by dependent issue, so more of them with two slots each beat fewer with three (decode of 64 contexts of 2600
// tokens on average at 8 x 128 / 128: 138-181 us with 7 x 2 against 164-201 us with 4 x 3; 4 x 96 / 64: 72 us with
// 8 x 2 against 106 us).
struct Shape { int warps, stages; };
Shape shape_of(int boxes) {
  switch (boxes) {
    case 2: return {12, 2};
    case 3: return {8, 2};
    case 4: return {7, 2};
    case 5: return {5, 2};
    case 6: return {4, 2};
    default: return {3, 2};
  }
}

template <int KB, int VB, bool TABLE>
b200_status launch_mma(const b200_kv* kv, WinArgs& a, int layer, cudaStream_t s) {
  const int boxes = (a.L.kd + 63) / 64 + (a.L.vd + 63) / 64;
  const Shape sh = shape_of(boxes);
  static_assert(most_warps(1, 1) >= 12 && most_warps(2, 1) >= 8 && most_warps(1, 2) >= 8, "a block's shape exceeds its launch bound");
  a.stages = sh.stages;
  const size_t smem = (size_t)sh.warps * sh.stages * (boxes * 4096 + sizeof(uint64_t)) + 1024;
  static bool configured = false;
  if (!configured) {
    B200_CUDA_TRY((cudaFuncSetAttribute(window_attn_mma_kernel<KB, VB, TABLE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024)));
    configured = true;
  }
  window_attn_mma_kernel<KB, VB, TABLE><<<g_sms, sh.warps * 32, smem, s>>>(kv->lay_kmap[layer], kv->lay_vmap[layer], a);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

template <int KB>
b200_status launch_mma_v(const b200_kv* kv, WinArgs& a, int layer, cudaStream_t s) {
  if (a.L.vd <= 64) return a.dist ? launch_mma<KB, 1, true>(kv, a, layer, s) : launch_mma<KB, 1, false>(kv, a, layer, s);
  if (a.L.vd <= 128) return a.dist ? launch_mma<KB, 2, true>(kv, a, layer, s) : launch_mma<KB, 2, false>(kv, a, layer, s);
  return a.dist ? launch_mma<KB, 4, true>(kv, a, layer, s) : launch_mma<KB, 4, false>(kv, a, layer, s);
}

}  // namespace

extern int b200_attn_pages_per_chunk;

b200_status b200_attn_make_plan(b200_kv* kv, int32_t window, int32_t qt, int32_t items_per_chunk, int32_t n_workers, const int32_t* d_row_seq,
                                const int32_t* d_row_ctx, int32_t total_rows, void* stream, float item_cost, float slot_cost, bool fine) {
  if (total_rows <= 0) return B200_OK;
  if (total_rows > kv->cfg.max_rows) { b200_set_error("attention: %d rows > max_rows %d", total_rows, kv->cfg.max_rows); return B200_ERR_CAPACITY; }
  const int R = kv->cfg.max_rows + 2;
  WindowPlan* p = find_plan(kv, window, qt, fine);
  if (!p) {
    p = new WindowPlan();
    p->window = window;
    p->q_tokens = qt;
    p->fine = fine;
    if (cudaMalloc((void**)&p->buf, sizeof(int) * ((size_t)5 * R + 4)) != cudaSuccess) {
      delete p;
      b200_set_error("attention plan: out of device memory");
      return B200_ERR_CUDA;
    }
    kv->plans.push_back(p);
  }
  const int forced = b200_attn_pages_per_chunk <= 0 ? 0 : std::min(std::max(b200_attn_pages_per_chunk, 1), 1 << 20);
  auto* kernel = fine ? window_plan_kernel<FineLengths> : window_plan_kernel<CoarseLengths>;
  kernel<<<1, 1024, 0, (cudaStream_t)stream>>>(d_row_seq, d_row_ctx, total_rows, kv->cfg.page_size, window, qt,
                                                          items_per_chunk, n_workers, forced, kv->max_chunks, item_cost, slot_cost,
                                                          p->buf, p->buf + R, p->buf + 2 * R, p->buf + 3 * R, p->buf + 4 * R, p->buf + 5 * R);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

bool b200_attn_use_plan(b200_kv* kv, int32_t window, int32_t q_tokens, bool fine, WinArgs* a) {
  const WindowPlan* p = find_plan(kv, window, q_tokens, fine);
  if (!p) { b200_set_error("attention: no plan for window %d and groups of %d", window, q_tokens); return false; }
  const int R = kv->cfg.max_rows + 2;
  a->group_first = p->buf; a->chunk_start = p->buf + R; a->part_base = p->buf + 2 * R; a->row_group = p->buf + 3 * R; a->page_base = p->buf + 4 * R;
  a->hdr = p->buf + 5 * R;
  a->part_o = kv->d_part_o; a->part_ml = kv->d_part_ml;
  return true;
}

b200_status b200_attn_combine(b200_kv* kv, const WinArgs& a, void* stream) {
  const long long rows = (long long)a.total_rows * a.n_q_heads;
  // few rows (decode): their columns over several blocks
  window_combine_kernel<<<dim3((unsigned)((rows + 7) / 8), rows <= 8192 ? (a.L.vd + 127) / 128 : 1), 256, 0, (cudaStream_t)stream>>>(a);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

b200_status b200_window_attn_plan(b200_kv* kv, int32_t layer, int32_t window, int32_t gqa, const int32_t* d_row_seq, const int32_t* d_row_ctx,
                                  int32_t total_rows, void* stream) {
  if (total_rows <= 0) return B200_OK;
  b200_status st = sm_count();
  if (st != B200_OK) return st;
  const KvLayerDev& L = kv->lay[layer];
  if (L.values_in_keys) return b200_latent_attn_plan(kv, layer, window, gqa, d_row_seq, d_row_ctx, total_rows, stream);
  const int per_chunk = L.heads * ((gqa + 15) / 16), warps = shape_of((L.kd + 63) / 64 + (L.vd + 63) / 64).warps;
  return b200_attn_make_plan(kv, window, q_tokens_of(gqa), per_chunk, g_sms * warps, d_row_seq, d_row_ctx, total_rows, stream, 1.25f, 0.25f, false);
}

b200_status b200_window_attn_run(b200_kv* kv, const WindowAttnCall& c, const int32_t* d_row_seq, const int32_t* d_row_ctx, int32_t total_rows,
                                 bool mma, void* stream) {
  if (c.layer < 0 || c.layer >= kv->cfg.n_layers || !kv->layered) { b200_set_error("window attention: layer %d of no layered pool", c.layer); return B200_ERR_INVALID_ARGUMENT; }
  const KvLayerDev& L = kv->lay[c.layer];
  if (L.heads <= 0 || c.n_q_heads <= 0 || c.n_q_heads % L.heads != 0) { b200_set_error("window attention: %d query heads over %d kv heads", c.n_q_heads, L.heads); return B200_ERR_INVALID_ARGUMENT; }
  if (total_rows <= 0) return B200_OK;
  if (total_rows > kv->cfg.max_rows) { b200_set_error("attention: %d rows > max_rows %d", total_rows, kv->cfg.max_rows); return B200_ERR_CAPACITY; }
  b200_status st = sm_count();
  if (st != B200_OK) return st;
  cudaStream_t s = (cudaStream_t)stream;
  const int G = c.n_q_heads / L.heads;
  if (!b200_window_attn_takes_mma(kv, c.layer) || !mma) {
    SimtArgs a;
    a.d = kv->dev; a.L = L; a.q = c.q; a.q_stride = c.q_stride; a.row_seq = d_row_seq; a.row_ctx = d_row_ctx; a.total_rows = total_rows;
    a.n_q_heads = c.n_q_heads; a.window = c.window; a.scale = c.scale; a.slopes_log2 = c.slopes_log2; a.sinks_log2 = c.sinks_log2;
    a.dist_log2 = c.dist_log2; a.dist_len = c.dist_len;
    a.out = c.out; a.out_stride = c.out_stride; a.out_head_stride = c.out_head_stride > 0 ? c.out_head_stride : L.value_dim;
    const size_t smem = sizeof(float) * 4 * (L.key_dim + L.value_dim);
    if (smem > 200 * 1024) { b200_set_error("window attention: head widths %d / %d are too large", L.key_dim, L.value_dim); return B200_ERR_UNSUPPORTED; }
    const unsigned grid = (unsigned)(((long long)total_rows * c.n_q_heads + 3) / 4);
    auto* kernel = kv->dev.elem_bytes == 4 ? attn_simt_kernel<float> : attn_simt_kernel<__nv_bfloat16>;
    if (smem > 48 * 1024) B200_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kernel<<<grid, 128, smem, s>>>(a);
    B200_LAUNCH_CHECK();
    return B200_OK;
  }
  if (L.values_in_keys) return b200_latent_attn_run(kv, c, d_row_seq, d_row_ctx, total_rows, stream);
  WinArgs a;
  if (!b200_attn_use_plan(kv, c.window, q_tokens_of(G), false, &a)) return B200_ERR_INVALID_ARGUMENT;
  a.d = kv->dev; a.L = L; a.q = (const __nv_bfloat16*)c.q; a.q_stride = c.q_stride; a.row_seq = d_row_seq; a.row_ctx = d_row_ctx;
  a.total_rows = total_rows; a.n_q_heads = c.n_q_heads; a.window = c.window;
  a.G = G; a.head_block = head_block_of(G); a.n_blocks = (G + 15) / 16;
  a.scale_log2 = c.scale * kLog2e;
  a.slopes = c.slopes_log2; a.sinks = c.sinks_log2; a.dist = c.dist_log2; a.dist_len = c.dist_len;
  a.out = (__nv_bfloat16*)c.out; a.out_stride = c.out_stride; a.out_head = c.out_head_stride > 0 ? c.out_head_stride : L.value_dim;
  if (L.kd <= 64) st = launch_mma_v<1>(kv, a, c.layer, s);
  else if (L.kd <= 128) st = launch_mma_v<2>(kv, a, c.layer, s);
  else st = launch_mma_v<4>(kv, a, c.layer, s);
  if (st != B200_OK) return st;
  // a window that spans no more pages than the shortest chunk the plan may choose never leaves partial sums
  const int shortest = b200_attn_pages_per_chunk > 0 ? b200_attn_pages_per_chunk : 4;
  const int most_pages = c.window > 0 ? (c.window + q_tokens_of(G) - 2) / 32 + 2 : kv->cfg.max_pages_per_seq;
  if (std::min(most_pages, kv->cfg.max_pages_per_seq) <= shortest) return B200_OK;
  return b200_attn_combine(kv, a, stream);
}

bool b200_window_attn_takes_mma(const b200_kv* kv, int32_t layer) {
  if (kv->layered && kv->lay[layer].values_in_keys) return b200_latent_attn_takes_mma(kv, layer);
  return kv->layered && kv->dev.elem_bytes == 2 && kv->lay[layer].kd <= 256 && kv->lay[layer].vd <= 256;
}
