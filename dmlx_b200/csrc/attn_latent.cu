// Latent attention: all heads attend to one row per token, [latent c | rotated key part], and their values are W_uv c.  W_uk is
// taken to the query side (q_head <- W_uk^T q_head) and W_uv behind the weighted sum, so the pages are read once for all heads
// and hold kv_rank + rot_dim numbers per token.
//
// latent_attn_kernel (tcgen05, bf16): half-tiles of 64 keys (two pages, one TMA box per 64 columns of a page) against up to 32 rows,
// a row being (token of the group, head).  The operands are swapped, so the keys fill the M side whatever the number of rows:
//   S^T [keys][rows] = K Q^T,          A = the keys as they lie (K-major), B = the rows' queries;
//   O^T [latent][rows] += C^T P,       A = the same keys read the other way (their latent columns are the M side), B = P.
// Even and odd half-tiles go through two groups of softmax warps with sums of their own, so that loads, products and softmax of
// neighbours overlap; the groups are added up at the end of a work item.  A thread holds one key and half of the rows; maxima over
// the keys go through a shuffle transpose, but only when some key exceeds a row's scale by 2^8 (then four correction warps, which
// reach all lanes of the sums, rescale them).  P enters the second product as two bf16 terms (value and remainder): weights keep
// 16 bits.
#include <cuda_bf16.h>

#include <algorithm>

#include "attn_latent.cuh"
#include "attn_plan.cuh"
#include "common.h"
#include "ptx.cuh"
#include "tma.cuh"

namespace {

// Angles in f64, brought into one turn before they become f32: positions far out keep their accuracy.
__global__ void __launch_bounds__(256) rotation_table_kernel(const double* __restrict__ freq, int half, float size, const int* __restrict__ pos, int rows,
                                                             float2* __restrict__ out) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= (long long)rows * half) return;
  const int row = (int)(i / half), p = (int)(i - (long long)row * half);
  constexpr double kTurn = 6.283185307179586476925286766559;
  const double a = (double)pos[row] * freq[p];
  float s, c;
  sincosf((float)(a - rint(a / kTurn) * kTurn), &s, &c);
  out[i] = make_float2(c * size, s * size);
}

struct PrepArgs {
  KvDev d;
  KvLayerDev L;
  LatentPrep p;
  const int *pos, *row_seq;
};

// One warp per (row, query head); blocks of their own for the row's latent and its query latent.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_prep_kernel(PrepArgs a) {
  const LatentPrep& p = a.p;
  __shared__ float part[32];
  const int row = blockIdx.x, lane = threadIdx.x & 31, head_blocks = (p.heads + 7) / 8, u = blockIdx.y * 8 + (threadIdx.x >> 5);
  const bool of_heads = (int)blockIdx.y < head_blocks;
  if (of_heads && u >= p.heads) return;
  const int per_head = p.dim + p.rot;
  const float2* rt = p.rotation + (size_t)row * (p.rot / 2);
  auto rotate = [&](T* dst, int col, int first, int step) {
    for (int i = first; i < p.rot / 2; i += step) {
      const int at = p.halves ? i : 2 * i, to = p.halves ? i + p.rot / 2 : 2 * i + 1;
      const float x = mat_value<T, 1>(p.src, row, col + at).v[0], y = mat_value<T, 1>(p.src, row, col + to).v[0];
      const float2 cs = rt[i];
      st(dst + at, x * cs.x - y * cs.y);
      st(dst + to, y * cs.x + x * cs.y);
    }
  };
  // by the whole block: columns col .. col + n - 1 divided by their root mean square, times w (the first ones stay in registers)
  auto normed = [&](T* dst, int col, int n, const float* w) {
    constexpr int KEEP = 2;
    Vec<VEC> keep[KEEP];
    float ss = 0.f;
    auto each = [&](auto f) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int c = (k * 256 + (int)threadIdx.x) * VEC;
        if (c < n) f(c, k);
      }
      for (int c = (KEEP * 256 + (int)threadIdx.x) * VEC; c < n; c += 256 * VEC) f(c, -1);
    };
    each([&](int c, int k) {
      const Vec<VEC> v = mat_value<T, VEC>(p.src, row, col + c);
      if (k >= 0) keep[k] = v;
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += v.v[e] * v.v[e];
    });
    const float r = 1.0f / sqrtf(block_sum(ss, part) / (float)n + p.eps);
    each([&](int c, int k) {
      Vec<VEC> v = k >= 0 ? keep[k >= 0 ? k : 0] : mat_value<T, VEC>(p.src, row, col + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] *= r * w[c + e];
      store_vec<VEC>(dst + c, v);
    });
  };
  if (of_heads) {
    T* plain = (T*)p.q_plain + ((size_t)row * p.heads + u) * p.plain_stride;
    for (int c = lane * VEC; c < p.dim; c += 32 * VEC) store_vec<VEC>(plain + c, mat_value<T, VEC>(p.src, row, u * per_head + c));
    for (int c = p.dim + lane; c < p.plain_stride; c += 32) st(plain + c, 0.f);
    T* q = (T*)p.q + ((size_t)row * p.heads + u) * a.L.kd;
    rotate(q + p.rank, u * per_head + p.dim, lane, 32);
    for (int c = a.L.key_dim + lane; c < a.L.kd; c += 32) st(q + c, 0.f);
    return;
  }
  if ((int)blockIdx.y > head_blocks || !p.keys) {
    if (p.q_rank == 0) return;
    T* dst = (T*)p.q_latent + (size_t)row * p.q_latent_stride;
    normed(dst, 0, p.q_rank, p.q_norm);
    for (int c = p.q_rank + (int)threadIdx.x; c < p.q_latent_stride; c += 256) st(dst + c, 0.f);
    return;
  }
  const int pos = a.pos[row], seq = a.row_seq[row];
  const int page_idx = pos / a.d.page_size, slot = pos - page_idx * a.d.page_size;
  // a step whose reservation failed has no page for this row: nothing is written (the error word is set)
  if (seq < 0 || seq >= a.d.max_seqs || page_idx >= a.d.seq_pages[seq]) return;
  const int page = a.d.block_table[(size_t)seq * a.d.max_pages_per_seq + page_idx];
  T* dst = (T*)((char*)a.d.k_pool + a.L.k_off) + ((size_t)page * a.d.page_size + slot) * (size_t)a.L.kd;
  const int col = p.q_rank + p.heads * per_head;
  normed(dst, col, p.rank, p.norm);
  rotate(dst + p.rank, col + p.rank, threadIdx.x, 256);
}

}  // namespace

b200_status b200_rotation_table(const double* d_freq, int dims, double size, const int32_t* d_pos, int rows, float2* d_out, void* stream) {
  if (rows <= 0 || dims < 2) return B200_OK;
  const long long n = (long long)rows * (dims / 2);
  rotation_table_kernel<<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(d_freq, dims / 2, (float)size, d_pos, rows, d_out);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

b200_status b200_latent_prep(b200_kv* kv, const LatentPrep& p, const int32_t* d_pos, const int32_t* d_row_seq, int rows, void* stream) {
  if (p.layer < 0 || p.layer >= kv->cfg.n_layers || !kv->layered || !kv->lay[p.layer].values_in_keys || kv->lay[p.layer].heads != 1 ||
      kv->lay[p.layer].key_dim != p.rank + p.rot || kv->lay[p.layer].value_dim != p.rank || p.rot % 2 != 0) {
    b200_set_error("latent attention: layer %d of the pool does not hold %d + %d numbers per token", p.layer, p.rank, p.rot);
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (rows <= 0) return B200_OK;
  PrepArgs a;
  a.d = kv->dev; a.L = kv->lay[p.layer]; a.p = p; a.pos = d_pos; a.row_seq = d_row_seq;
  const bool v4 = p.dim % 4 == 0 && p.rot % 4 == 0 && p.rank % 4 == 0 && p.plain_stride % 4 == 0 && p.q_rank % 4 == 0 && p.q_latent_stride % 4 == 0 && (p.src.ws || p.src.y_stride % 4 == 0);
  auto* kernel = kv->dev.elem_bytes == 4 ? (v4 ? latent_prep_kernel<float, 4> : latent_prep_kernel<float, 1>)
                                         : (v4 ? latent_prep_kernel<__nv_bfloat16, 4> : latent_prep_kernel<__nv_bfloat16, 1>);
  kernel<<<dim3(rows, (p.heads + 7) / 8 + (p.keys ? 1 : 0) + (p.q_rank > 0 ? 1 : 0)), 256, 0, (cudaStream_t)stream>>>(a);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

// ---- tensor-core kernel ----------------------------------------------------------------------------------------------
namespace {

// A stage of the ring holds two half-tiles of 64 keys (two pages) per 64-column box, one behind the other, so that a product with
// M = 128 can read either: its other 64 rows are then whatever lies in the other half, in tensor-memory lanes nobody reads.
constexpr int kHalfKeys = 64, kHalfPages = 2, kHalfBytes = kHalfKeys * 128, kBoxBytes = 2 * kHalfBytes;
constexpr int kPBytes = kHalfKeys * 128;
constexpr int kLatentThreads = 512;    // warp 0 loads, warp 1 issues the MMAs, warps 4-11 softmax, 12-15 correction
constexpr int kMaxStages = 4;
constexpr float kGrow = 8.f;           // log2 units a row's maximum may grow before its sums are rescaled
constexpr uint32_t kPolls = 1u << 18;  // a wait inside a CTA is microseconds

__device__ __forceinline__ bool wait(uint64_t* bar, uint32_t parity) { return ptx::mbar_wait_limit(bar, parity, kPolls); }
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void bar_sync(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
// ... and whether some thread passed true.
__device__ __forceinline__ bool bar_any(int id, int threads, bool x) {
  uint32_t r;
  asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.b32 p, %1, 0;\n\tbar.red.or.pred q, %2, %3, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
               : "=r"(r) : "r"((uint32_t)x), "r"(id), "r"(threads) : "memory");
  return r != 0;
}

// Reduces N values over the warp's lanes: every step hands half of the columns to the partner lane.  Lane l ends up with
// column l / (32 / N).
template <int N, bool MAX>
__device__ __forceinline__ float transpose_reduce(float (&w)[N], int lane) {
  int o = 16;
#pragma unroll
  for (int n = N / 2; n >= 1; n >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float send = up ? w[i] : w[i + n], keep = up ? w[i + n] : w[i];
      const float got = __shfl_xor_sync(0xffffffffu, send, o);
      w[i] = MAX ? fmaxf(keep, got) : keep + got;
    }
    o >>= 1;
  }
#pragma unroll
  for (int b = 16 / N; b >= 1; b >>= 1) {
    const float got = __shfl_xor_sync(0xffffffffu, w[0], b);
    w[0] = MAX ? fmaxf(w[0], got) : w[0] + got;
  }
  return w[0];
}

template <int N>
__device__ __forceinline__ void tmem_load(uint32_t taddr, uint32_t (&u)[N]) {
  if constexpr (N == 8) ptx::tmem_ld8(taddr, u);
  else ptx::tmem_ld16(taddr, u);
}
template <int N>
__device__ __forceinline__ void tmem_store(uint32_t taddr, const uint32_t (&u)[N]) {
  if constexpr (N == 8) ptx::tmem_st8(taddr, u);
  else ptx::tmem_st16(taddr, u);
}

struct LatentArgs {
  WinArgs w;
  int n_kb, n_mc;     // 64-column boxes of a key row; blocks of 128 latent columns
  uint32_t tmem_cols;
};

// Shared memory behind the tiles, the queries and P.  [2]: half-tiles with an even and an odd number, which the two groups of
// softmax warps take.
template <int NR>
struct LatentShared {
  uint64_t k_full[kMaxStages][2], k_free[kMaxStages][2], s_full[2][2], p_ready[2], pv_done[2], c_req[2], c_done[2], q_full, q_free;
  long long off[NR];  // where a row's output starts (-1: the row does not exist)
  WinItem items[2];   // the loading thread looks an item up for everyone
  int3 range;         // the block's work items
  uint32_t tmem;
  int done;
  float red[2][2][NR], m[2][NR], corr[2][NR], w[2][NR];
  int ctx[NR], lo[NR];  // a row sees keys lo .. ctx - 1
};

template <int NR>
__global__ void __launch_bounds__(kLatentThreads, 1)
    latent_attn_kernel(const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap qmap, LatentArgs la) {
  const WinArgs& a = la.w;
  extern __shared__ unsigned char latent_dyn[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(latent_dyn) + 1023) & ~(uintptr_t)1023);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, stages = a.stages, n_kb = la.n_kb, n_mc = la.n_mc;
  const int stage_bytes = n_kb * kBoxBytes;
  unsigned char* qbuf = smem + (size_t)stages * stage_bytes;  // [box][NR rows][128 B]
  unsigned char* pbuf = qbuf + (size_t)n_kb * NR * 128;       // [group][values, remainders][key][128 B, NR of 64 columns used]
  LatentShared<NR>& sh = *reinterpret_cast<LatentShared<NR>*>(pbuf + 4 * kPBytes);
  const int n_groups = a.hdr[0];
  if (tid == 0) {
    for (int h = 0; h < 2; ++h) {
      for (int s = 0; s < stages; ++s) { ptx::mbar_init(&sh.k_full[s][h], 1); ptx::mbar_init(&sh.k_free[s][h], 1); }
      ptx::mbar_init(&sh.s_full[h][0], 1);
      ptx::mbar_init(&sh.s_full[h][1], 1);
      ptx::mbar_init(&sh.p_ready[h], 128);
      ptx::mbar_init(&sh.pv_done[h], 1);
      ptx::mbar_init(&sh.c_req[h], 1);
      ptx::mbar_init(&sh.c_done[h], 128);
    }
    ptx::mbar_init(&sh.q_full, 1);
    ptx::mbar_init(&sh.q_free, 1);
    ptx::mbar_fence_init();
    sh.done = 0;
    sh.range = worker_items(a, n_groups);
  }
  if (warp == 1) {
    ptx::tmem_alloc(&sh.tmem, la.tmem_cols);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before_sync();
  __syncthreads();
  ptx::tc_fence_after_sync();
  const int item0 = sh.range.x, n_items = sh.range.y, item_step = sh.range.z;
  const uint32_t tmem = sh.tmem, tmem_o = tmem + 4 * NR;  // S of the two groups, twice each, then O of the two: n_mc x NR columns each
  bool ok = true;

  if (warp == 0) {
    if (lane == 0) {  // ---- loads ----
      int s = 0;
      uint32_t used = 0, phase = 0, n_item = 0;  // bit 2 * stage + half: loaded before; parity of its next load
      // Looking an item up takes a chain of dependent loads: it is done while the item before is being worked on.
      WinItem ahead{};
      int next[kHalfPages], ahead_id[kHalfPages];  // page ids of the coming half-tile, and of the coming item's first
      auto look_up = [&](int item) {
        if (item >= n_items) return;
        ahead = decode_item(a, item, n_groups);
        const int* table = a.d.block_table + (size_t)ahead.seq * a.d.max_pages_per_seq;
#pragma unroll
        for (int p = 0; p < kHalfPages; ++p) ahead_id[p] = ahead.page_begin + p < ahead.page_end ? table[ahead.page_begin + p] : 0;
      };
      look_up(item0);
      for (int item = item0; item < n_items && ok; item += item_step, ++n_item) {
        const WinItem it = ahead;
        const int* table = a.d.block_table + (size_t)it.seq * a.d.max_pages_per_seq;
#pragma unroll
        for (int p = 0; p < kHalfPages; ++p) next[p] = ahead_id[p];
        bool looked = false;
        ok = wait(&sh.q_free, (n_item & 1u) ^ 1u);
        if (!ok) break;
        sh.items[n_item & 1u] = it;
        // the tile's rows lie one behind the other: tokens of the group, or heads of the block (what follows them is never stored)
        ptx::mbar_expect_tx(&sh.q_full, n_kb * NR * 128);
        for (int b = 0; b < n_kb; ++b)
          ptx::tma_load_2d(qbuf + b * NR * 128, &qmap, b * 64, it.first_row * a.n_q_heads + it.block * a.head_block, &sh.q_full);
        int h = 0;
        for (int pg = it.page_begin; pg < it.page_end; pg += kHalfPages) {
          const int pages = min(kHalfPages, it.page_end - pg), slot = 2 * s + h;
          if (pg == it.page_begin + 2 * kHalfPages) { look_up(item + item_step); looked = true; }
          int id[kHalfPages];
#pragma unroll
          for (int p = 0; p < kHalfPages; ++p) {
            id[p] = next[p];
            const int later = pg + kHalfPages + p;
            next[p] = later < it.page_end ? table[later] : 0;
          }
          ok = wait(&sh.k_free[s][h], ((phase >> slot) & 1u) ^ 1u);
          if (!ok) break;
          ptx::mbar_expect_tx(&sh.k_full[s][h], pages * n_kb * 4096);
          unsigned char* dst = smem + (size_t)s * stage_bytes + h * kHalfBytes;
          for (int b = 0; b < n_kb; ++b)
            for (int p = 0; p < pages; ++p) ptx::tma_load_2d(dst + b * kBoxBytes + p * 4096, &kmap, b * 64, id[p] * 32, &sh.k_full[s][h]);
          used |= 1u << slot;
          phase ^= 1u << slot;
          h ^= 1;
          if (h == 0 && ++s == stages) s = 0;
        }
        if (h == 1 && ++s == stages) s = 0;  // an item starts on an even half-tile
        if (!looked) look_up(item + item_step);
      }
      if (!ok) {  // leave no copy in flight behind
        if (n_item > 0) wait(&sh.q_full, (n_item - 1) & 1u);
        for (int slot = 0; slot < 2 * stages; ++slot)
          if (used >> slot & 1u) wait(&sh.k_full[slot >> 1][slot & 1], ((phase >> slot) & 1u) ^ 1u);
      }
    }
  } else if (warp == 1) {
    if (ptx::elect_one()) {  // ---- matrix products ----
      const uint32_t id_s = ptx::umma_idesc_bf16(128, NR), id_o = id_s | ptx::kUmmaAMn | ptx::kUmmaBMn;
      // descriptors advance by adding to their address field (16-byte units)
      const uint64_t q_desc = ptx::umma_desc_k_sw128(ptx::smem_u32(qbuf)), k_desc = ptx::umma_desc_k_sw128(ptx::smem_u32(smem));
      const uint64_t v_desc = ptx::umma_desc_mn_sw128(ptx::smem_u32(smem), kBoxBytes), p_desc = ptx::umma_desc_mn_sw128(ptx::smem_u32(pbuf), kPBytes);
      int s0 = 0;  // stage of the item's first half-tile
      uint32_t phase = 0, n_item = 0, n_p[2] = {0, 0}, n_sc[2] = {0, 0};
      for (int item = item0; item < n_items && ok; item += item_step, ++n_item) {
        ok = wait(&sh.q_full, n_item & 1u);
        if (!ok) break;
        const int n_pages = sh.items[n_item & 1u].page_end - sh.items[n_item & 1u].page_begin, halves = (n_pages + kHalfPages - 1) / kHalfPages;
        int scored = 0, summed = 0, ss = s0, ps = s0;  // half-tiles, and the stages of the next ones
        uint32_t idle = 0;
        // whichever of the two next products has its operands goes first
        while (summed < halves) {
          const int hs = scored & 1, hp = summed & 1, slot = 2 * ss + hs;
          if (scored < halves && scored < summed + 4 && ptx::mbar_test(&sh.k_full[ss][hs], (phase >> slot) & 1u)) {
            ptx::tc_fence_after_sync();
            const uint64_t k0 = k_desc + (uint64_t)(ss * (stage_bytes >> 4));
            const uint32_t buf = n_sc[hs]++ & 1u, dst = tmem + (2 * hs + buf) * NR;
            for (int b = 0; b < n_kb; ++b) {  // (columns behind the row's width are zeros)
              const uint64_t da = k0 + (uint64_t)(b * (kBoxBytes >> 4)), db = q_desc + (uint64_t)(b * (NR * 128 >> 4));
#pragma unroll
              for (int k4 = 0; k4 < 4; ++k4) ptx::umma_bf16(dst, da + 2 * k4, db + 2 * k4, id_s, b + k4 > 0 ? 1u : 0u);
            }
            ptx::umma_commit(&sh.s_full[hs][buf]);
            phase ^= 1u << slot;
            ++scored;
            if (scored == halves) ptx::umma_commit(&sh.q_free);
            if (hs == 1 && ++ss == stages) ss = 0;
            idle = 0;
          } else if (summed < scored && ptx::mbar_test(&sh.p_ready[hp], n_p[hp] & 1u)) {
            ptx::tc_fence_after_sync();
            const int pages = min(kHalfPages, n_pages - summed * kHalfPages);
            const uint64_t v0 = v_desc + (uint64_t)(ps * (stage_bytes >> 4) + hp * (kHalfBytes >> 4)), p0 = p_desc + (uint64_t)(hp * (2 * kPBytes >> 4));
            for (int mc = 0; mc < n_mc; ++mc) {
              const uint32_t dst = tmem_o + (hp * n_mc + mc) * NR;
              for (int pg = 0; pg < pages; ++pg) {
                const uint64_t va = v0 + (uint64_t)(mc * (2 * kBoxBytes >> 4) + pg * (4096 >> 4)), pb = p0 + (uint64_t)(pg * (4096 >> 4));
#pragma unroll
                for (int ks = 0; ks < 2; ++ks) {
                  ptx::umma_bf16(dst, va + ks * (2048 >> 4), pb + ks * (2048 >> 4), id_o, summed > 1 || pg + ks > 0 ? 1u : 0u);
                  ptx::umma_bf16(dst, va + ks * (2048 >> 4), pb + ((kPBytes + ks * 2048) >> 4), id_o, 1u);
                }
              }
            }
            ptx::umma_commit(&sh.k_free[ps][hp]);
            ptx::umma_commit(&sh.pv_done[hp]);
            ++n_p[hp];
            ++summed;
            if (hp == 1 && ++ps == stages) ps = 0;
            idle = 0;
          } else if (++idle > (1u << 26)) {
            ok = false;
            break;
          }
        }
        s0 += (halves + 1) / 2 % stages;
        if (s0 >= stages) s0 -= stages;
      }
    }
  } else if (warp >= 4 && warp < 12) {
    // ---- softmax: group 0 takes the even half-tiles, group 1 the odd ones; thread = (key = tensor-memory lane, half of the rows) ----
    constexpr int NC = NR / 2, kAll = 3, kAllThreads = 256;
    const int quarter = warp & 3, g = quarter >> 1, key = (quarter & 1) * 32 + lane, c0 = warp >= 8 ? NC : 0;
    const int row = (warp >= 8 ? 64 : 0) + key;  // thread of the group; row < NR: it keeps that row
    const uint32_t lanes = (uint32_t)(quarter * 32) << 16;
    const int hb = a.head_block;
    unsigned char* p_hi = pbuf + g * 2 * kPBytes + key * 128;
    uint32_t n_s = 0, n_pv = 0, n_c = 0, n_item = 0;  // half-tiles of the group scored / summed, rescalings, items (phases of the barriers)
    bool dead = false;                       // some thread's wait ran out: decided together, so that all leave
    for (int item = item0; item < n_items; item += item_step, ++n_item) {
      // (not q_full: that barrier may be two phases on when the item before is still being written out)
      if (g == 0) ok = wait(&sh.s_full[0][n_s & 1u], (n_s >> 1) & 1u) && ok;
      if (bar_any(kAll, kAllThreads, !ok)) { dead = true; break; }
      const WinItem it = sh.items[n_item & 1u];
      const int h0 = it.block * hb, heads_here = min(hb, a.n_q_heads - h0), n_pages = it.page_end - it.page_begin;
      const int halves = (n_pages + kHalfPages - 1) / kHalfPages;
      const int lo_last = first_key(it.ctx0 + it.n_rows - 1, a.window);  // the latest window start of the group
      if (row < NR) {
        if (g == 0) {
          const int tok = row / hb, head = row - tok * hb;
          const bool on = tok < it.n_rows && head < heads_here;
          sh.ctx[row] = on ? it.ctx0 + tok : 0;
          sh.lo[row] = first_key(sh.ctx[row], a.window);
          sh.off[row] = !on ? -1 : it.slot0 >= 0 ? ((long long)(it.slot0 + tok) * a.n_q_heads + h0 + head) * a.L.vd
                                      : (long long)(it.first_row + tok) * a.out_stride + (long long)(h0 + head) * a.out_head;
        }
        sh.m[g][row] = kAttnNone;
      }
      float l[NC], m[NC];
#pragma unroll
      for (int r = 0; r < NC; ++r) { l[r] = 0.f; m[r] = kAttnNone; }
      bar_sync(kAll, kAllThreads);
      bool broken = false;
      for (int j = g; j < halves; j += 2) {
        const int pages = min(kHalfPages, n_pages - j * kHalfPages), tok0 = (it.page_begin + j * kHalfPages) * 32;
        const bool first = j == g;
        ok = wait(&sh.s_full[g][n_s & 1u], (n_s >> 1) & 1u) && ok;
        const uint32_t s_at = tmem + lanes + (2 * g + (n_s & 1u)) * NR + c0;
        ++n_s;
        ptx::tc_fence_after_sync();
        __syncwarp();
        float v[NC];
        {
          uint32_t u[NC];
          tmem_load<NC>(s_at, u);
          ptx::tmem_ld_wait();
#pragma unroll
          for (int r = 0; r < NC; ++r) v[r] = __uint_as_float(u[r]) * a.scale_log2;
        }
        if (tok0 + kHalfKeys > it.ctx0 || pages < kHalfPages || tok0 < lo_last) {
          const bool in_tile = key < pages * 32;
#pragma unroll
          for (int r = 0; r < NC; ++r) v[r] = in_tile && tok0 + key < sh.ctx[c0 + r] && tok0 + key >= sh.lo[c0 + r] ? v[r] : kAttnNone;
        }
        // The scale of a row stays as it is unless some key exceeds it by 2^kGrow; only then are the maxima taken.
        bool over = !ok;
#pragma unroll
        for (int r = 0; r < NC; ++r) over = over || v[r] > m[r] + kGrow;
        const bool move = bar_any(1 + g, 128, over);
        if (!first) {  // P and O are the previous half-tile's until its product is done
          ok = wait(&sh.pv_done[g], n_pv & 1u) && ok;
          ++n_pv;
          ptx::tc_fence_after_sync();
          __syncwarp();
        }
        if (move) {
          {
            float w[NC];
#pragma unroll
            for (int r = 0; r < NC; ++r) w[r] = v[r];
            const float mx = transpose_reduce<NC, true>(w, lane);
            if (lane % (32 / NC) == 0) sh.red[g][quarter & 1][c0 + lane / (32 / NC)] = mx;
          }
          if (bar_any(1 + g, 128, !ok)) { broken = true; break; }
          if (row < NR) {
            const float m_old = sh.m[g][row], mx = fmaxf(sh.red[g][0][row], sh.red[g][1][row]);
            const bool moved = mx > m_old + kGrow;
            sh.corr[g][row] = moved ? ex2(m_old - mx) : 1.f;
            if (moved) sh.m[g][row] = mx;
          }
          bar_sync(1 + g, 128);
          float corr[NC];
#pragma unroll
          for (int r = 0; r < NC; ++r) { corr[r] = sh.corr[g][c0 + r]; m[r] = sh.m[g][c0 + r]; l[r] *= corr[r]; }
          if (!first) {  // the sums lie in all 128 lanes, half of which this group's warps cannot reach
            ptx::tc_fence_before_sync();
            if (row == 0) ptx::mbar_arrive(&sh.c_req[g]);
            ok = wait(&sh.c_done[g], n_c & 1u) && ok;
            ++n_c;
            ptx::tc_fence_after_sync();
            __syncwarp();
          }
        }
#pragma unroll
        for (int r = 0; r < NC; r += 8) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float p[2];
#pragma unroll
            for (int f = 0; f < 2; ++f) {
              const int i = r + 2 * e + f;
              p[f] = v[i] > kAttnNone ? ex2(v[i] - m[i]) : 0.f;
              l[i] += p[f];
            }
            const __nv_bfloat162 h2 = __floats2bfloat162_rn(p[0], p[1]);
            const float2 back = __bfloat1622float2(h2);
            const __nv_bfloat162 l2 = __floats2bfloat162_rn(p[0] - back.x, p[1] - back.y);
            hi[e] = *reinterpret_cast<const uint32_t*>(&h2);
            lo[e] = *reinterpret_cast<const uint32_t*>(&l2);
          }
          const int at = ((((c0 + r) / 8) ^ (key & 7)) << 4);
          *reinterpret_cast<uint4*>(p_hi + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(p_hi + kPBytes + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
        ptx::fence_proxy_async_smem();
        ptx::tc_fence_before_sync();
        ptx::mbar_arrive(&sh.p_ready[g]);
      }
      if (!broken && g < halves) {
        ok = wait(&sh.pv_done[g], n_pv & 1u) && ok;
        ++n_pv;
      }
      {
        const float sum = transpose_reduce<NC, false>(l, lane);
        if (lane % (32 / NC) == 0) sh.red[g][quarter & 1][c0 + lane / (32 / NC)] = sum;
      }
      if (bar_any(kAll, kAllThreads, !ok)) { dead = true; break; }
      ptx::tc_fence_after_sync();
      if (g == 0 && row < NR && sh.ctx[row] > 0) {
        // the two groups' sums at a common scale
        const float m0 = sh.m[0][row], m1 = sh.m[1][row], mr = fmaxf(m0, m1);
        float w0 = ex2(m0 - mr), w1 = ex2(m1 - mr);
        float sum = w0 * (sh.red[0][0][row] + sh.red[0][1][row]) + w1 * (sh.red[1][0][row] + sh.red[1][1][row]);
        const int tok = row / hb, head = row - tok * hb;
        if (it.slot0 < 0) {
          float f = 1.f;
          if (a.sinks) {
            const float sk = a.sinks[h0 + head], mm = fmaxf(mr, sk);
            f = exp2f(mr - mm);
            sum = sum * f + exp2f(sk - mm);
          }
          const float inv = sum > 0.f ? f / sum : 0.f;
          w0 *= inv;
          w1 *= inv;
        } else {
          const size_t pidx = (size_t)(it.slot0 + tok) * a.n_q_heads + h0 + head;
          a.part_ml[pidx * 2] = mr;
          a.part_ml[pidx * 2 + 1] = sum;
        }
        sh.w[0][row] = w0;
        sh.w[1][row] = w1;
      }
      bar_sync(kAll, kAllThreads);
      for (int mc = 0; mc < n_mc; ++mc) {
        uint32_t o[NC], odd[NC];
        tmem_load<NC>(tmem_o + lanes + mc * NR + c0, o);
        if (halves > 1) tmem_load<NC>(tmem_o + lanes + (n_mc + mc) * NR + c0, odd);
        ptx::tmem_ld_wait();
        const int dim = mc * 128 + quarter * 32 + lane;
        // (shared memory is read ahead of the stores: the compiler cannot tell that they do not touch it)
        float x[NC];
#pragma unroll
        for (int r = 0; r < NC; ++r) x[r] = __uint_as_float(o[r]) * sh.w[0][c0 + r];
        if (halves > 1) {
#pragma unroll
          for (int r = 0; r < NC; ++r) x[r] = fmaf(__uint_as_float(odd[r]), sh.w[1][c0 + r], x[r]);
        }
        long long off[NC];
#pragma unroll
        for (int r = 0; r < NC; ++r) off[r] = sh.off[c0 + r];
        if (it.slot0 >= 0) {
#pragma unroll
          for (int r = 0; r < NC; ++r)
            if (off[r] >= 0 && dim < a.L.vd) a.part_o[off[r] + dim] = x[r];
        } else {
#pragma unroll
          for (int r = 0; r < NC; ++r)
            if (off[r] >= 0 && dim < a.L.value_dim) a.out[off[r] + dim] = __float2bfloat16(x[r]);
        }
        __syncwarp();
      }
      ptx::tc_fence_before_sync();
      bar_sync(kAll, kAllThreads);  // the item's shared values have been read
    }
    ok = ok && !dead;
    if (g == 0 && row == 0) *(volatile int*)&sh.done = 1;
  }
  if (warp >= 12) {
    // ---- correction: rescales a group's sums when one of its rows' scales has moved ----
    const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
    uint32_t n_c[2] = {0, 0}, idle = 0;
    bool go = true;
    while (go) {
      int what = -1;
      if (lane == 0) {
        const bool done = *(volatile int*)&sh.done != 0;  // (before the requests: none comes after it)
        for (int g = 0; g < 2 && what < 0; ++g)
          if (ptx::mbar_test(&sh.c_req[g], n_c[g] & 1u)) what = g;
        if (what < 0 && (done || ++idle > (1u << 24))) what = done ? 2 : 3;
      }
      what = __shfl_sync(0xffffffffu, what, 0);
      if (what >= 2) {
        ok = what == 2;
        break;
      }
      if (what < 0) {
        __nanosleep(100);
        continue;
      }
      const int g = what;
      ++n_c[g];
      idle = 0;
      ptx::tc_fence_after_sync();
      for (int mc = 0; mc < n_mc; ++mc) {
        for (int c = 0; c < NR; c += 16) {
          uint32_t o[16];
          const uint32_t at = tmem_o + lanes + (g * n_mc + mc) * NR + c;
          ptx::tmem_ld16(at, o);
          ptx::tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * sh.corr[g][c + e]);
          ptx::tmem_st16(at, o);
        }
      }
      ptx::tmem_st_wait();
      ptx::tc_fence_before_sync();
      ptx::mbar_arrive(&sh.c_done[g]);
    }
  }
  if (!ok) atomicExch(a.d.state + ST_ATTN_ERR, B200_ERR_DEVICE_FLAGGED);
  ptx::tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) ptx::tmem_dealloc(tmem, la.tmem_cols);
}

int g_sms = 0;
constexpr int kSmemLimit = 227 * 1024;

template <int NR>
size_t smem_of(int n_kb, int stages) {
  return (size_t)stages * n_kb * kBoxBytes + (size_t)n_kb * NR * 128 + 4 * kPBytes + sizeof(LatentShared<NR>) + 1024;
}

// Rows of a tile: 16 where a decode step would leave more of them empty, or where the keys leave no room for 32.
int rows_of(const KvLayerDev& L, int heads, int total_rows) {
  return (heads <= 16 && total_rows <= 256) || smem_of<32>((L.kd + 63) / 64, 1) > kSmemLimit ? 16 : 32;
}

template <int NR>
b200_status launch(const b200_kv* kv, LatentArgs& la, int layer, cudaStream_t s) {
  CUtensorMap qmap;
  const uint64_t dims[2] = {(uint64_t)la.w.L.kd, (uint64_t)la.w.total_rows * la.w.n_q_heads}, strides[1] = {(uint64_t)la.w.L.kd * 2};
  const uint32_t box[2] = {64, (uint32_t)NR};
  b200_status st = b200_make_tensor_map(&qmap, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, la.w.q, dims, strides, box);
  if (st != B200_OK) return st;
  int stages = kMaxStages;
  while (stages > 1 && smem_of<NR>(la.n_kb, stages) > kSmemLimit) --stages;
  la.w.stages = stages;
  la.tmem_cols = 32;
  while (la.tmem_cols < (uint32_t)(4 * NR + 2 * la.n_mc * NR)) la.tmem_cols <<= 1;
  static bool configured = false;
  if (!configured) {
    B200_CUDA_TRY(cudaFuncSetAttribute(latent_attn_kernel<NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit));
    configured = true;
  }
  latent_attn_kernel<NR><<<g_sms, kLatentThreads, smem_of<NR>(la.n_kb, stages), s>>>(kv->lay_kmap[layer], qmap, la);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

}  // namespace

bool b200_latent_attn_takes_mma(const b200_kv* kv, int32_t layer) {
  const KvLayerDev& L = kv->lay[layer];
  return kv->layered && L.values_in_keys && L.heads == 1 && kv->dev.elem_bytes == 2 && smem_of<16>((L.kd + 63) / 64, 1) <= kSmemLimit &&
         128 + (L.value_dim + 127) / 128 * 64 <= 512;
}

b200_status b200_latent_attn_plan(b200_kv* kv, int32_t layer, int32_t window, int32_t heads, const int32_t* d_row_seq, const int32_t* d_row_ctx, int32_t total_rows,
                                  void* stream) {
  if (g_sms == 0) {
    int dev = 0;
    B200_CUDA_TRY(cudaGetDevice(&dev));
    B200_CUDA_TRY(cudaDeviceGetAttribute(&g_sms, cudaDevAttrMultiProcessorCount, dev));
  }
  const int rows = rows_of(kv->lay[layer], heads, total_rows);
  return b200_attn_make_plan(kv, window, std::max(1, rows / heads), (heads + rows - 1) / rows, g_sms, d_row_seq, d_row_ctx, total_rows, stream, 4.f,
                             4.f * std::min(heads, rows) * kv->lay[layer].value_dim / (64.f * kv->lay[layer].kd), true);
}

b200_status b200_latent_attn_run(b200_kv* kv, const WindowAttnCall& c, const int32_t* d_row_seq, const int32_t* d_row_ctx, int32_t total_rows,
                                 void* stream) {
  const KvLayerDev& L = kv->lay[c.layer];
  if (c.q_stride != c.n_q_heads * L.kd) { b200_set_error("latent attention: query rows have to lie one behind the other"); return B200_ERR_INVALID_ARGUMENT; }
  if (c.slopes_log2) { b200_set_error("latent attention has no distance bias"); return B200_ERR_UNSUPPORTED; }
  LatentArgs la;
  WinArgs& a = la.w;
  const int rows = rows_of(L, c.n_q_heads, total_rows), hb = std::min(c.n_q_heads, rows);
  if (!b200_attn_use_plan(kv, c.window, std::max(1, rows / c.n_q_heads), true, &a)) return B200_ERR_INVALID_ARGUMENT;
  a.d = kv->dev; a.L = L; a.L.vd = (L.value_dim + 15) / 16 * 16;
  a.q = (const __nv_bfloat16*)c.q; a.q_stride = c.q_stride; a.row_seq = d_row_seq; a.row_ctx = d_row_ctx;
  a.total_rows = total_rows; a.n_q_heads = c.n_q_heads; a.window = c.window;
  a.G = c.n_q_heads; a.head_block = hb; a.n_blocks = (c.n_q_heads + hb - 1) / hb;
  a.scale_log2 = c.scale * kAttnLog2e;
  a.slopes = nullptr; a.sinks = c.sinks_log2;
  a.out = (__nv_bfloat16*)c.out; a.out_stride = c.out_stride; a.out_head = c.out_head_stride > 0 ? c.out_head_stride : L.value_dim;
  la.n_kb = (L.kd + 63) / 64;
  la.n_mc = (L.value_dim + 127) / 128;
  b200_status st = rows == 16 ? launch<16>(kv, la, c.layer, (cudaStream_t)stream) : launch<32>(kv, la, c.layer, (cudaStream_t)stream);
  if (st != B200_OK) return st;
  return b200_attn_combine(kv, a, stream);
}
