// Gated linear attention: per head a state S [dk][dv] in f32, S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t, with a decay per
// key channel; the state lives in the pool's slot of the sequence and is carried from step to step.  A sequence at position 0
// starts from zero, so slots need no clearing.
//
// gla_step_kernel: token by token, one CTA per (request, head): decay, state update, output, per-head norm and gate in one pass
// over the state (decode, short portions, f32).
//
// Longer portions go in chunks of 32 tokens.  With L_t the sum of log alpha since the chunk's start,
//   o_t = S_0^T (q_t e^{L_t}) + sum_{j <= t} (q_t . k_j e^{L_t - L_j}) v_j,   S_C = diag(e^{L_C}) S_0 + sum_j (k_j e^{L_C - L_j}) v_j^T.
//   gla_chunk_kernel  (chunk, head), all in parallel: decays, the scaled q and k, and the 32 x 32 weights of the sum;
//   gla_scan_kernel   (request, head, slice of dv): walks the chunks with S^T in registers, mma.sync;
//   gla_out_kernel    norm and gate of the rows.
// f32 factors enter the tensor cores as two bf16 terms (value and remainder); the state itself stays f32.
//
// Matrix memory runs through the same kernels: with the running maximum m taken out, S <- e^(f + m' - m) S + (e^(i - m) k) v^T has one
// decay per head and token, both factors at most 1, and the sum of the keys is one more value column whose values are ones.
// The delta rule (delta.cu) goes through the scan and out kernels, with more to do per chunk.
// memory_gates_kernel makes the factors (m is a scan over (max, +)); memory_chunk_kernel and memory_out_kernel take the places of the
// chunk and out kernels.
#include <cuda_bf16.h>

#include <algorithm>

#include "common.h"
#include "gla_chunks.cuh"

namespace {

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu(float g) { return g / (1.0f + expf(-g)); }
__device__ __forceinline__ float sigmoid(float g) { return 1.0f / (1.0f + expf(-g)); }
// Values of a matrix memory: columns dv and on are {1, 0, 0, ..}.
template <typename T, int VEC>
__device__ __forceinline__ Vec<VEC> memory_value(const Gla& a, int row, int head, int c) {
  if (c < a.dv) return mat_value<T, VEC>(a.src, row, a.col_v() + head * a.dv + c);  // (VEC divides dv)
  Vec<VEC> v{};
  v.v[0] = c == a.dv ? 1.f : 0.f;
  return v;
}

// ---- token by token ------------------------------------------------------------------------------------------
template <typename T, int VEC, bool MEM>
__global__ void __launch_bounds__(256, 3) gla_step_kernel(Gla a) {
  extern __shared__ float sh[];
  __shared__ float part[32];
  const int req = blockIdx.x, head = blockIdx.y, dk = a.dk, dv = a.dv, dvs = MEM ? a.dvs : dv, dva = MEM && VEC == 1 ? a.dva : dvs;
  const int r0 = a.cu[req], count = a.cu[req + 1] - r0;
  if (count <= 0 || (a.chunked && count > kGlaStepTokens) || a.d.state[ST_ERR] != 0) return;
  float *q = sh, *k = q + dk, *al = k + dk, *a1 = al + dk, *red = a1 + (MEM ? 0 : a.rank);  // red [groups][dvs]
  const int tid = threadIdx.x, nthr = blockDim.x, groups = a.groups, tx = tid % a.cols, ty = tid / a.cols;
  const int slot = a.row_seq[r0];
  if (slot < 0 || slot >= a.d.max_seqs) return;
  float* S = a.state + (size_t)slot * a.rec_elems + (size_t)head * dk * dvs;
  for (int t = 0; t < count; ++t) {
    const int row = r0 + t;
    const bool fresh = a.pos[row] == 0;
    float4 gate{};
    if constexpr (MEM) {
      gate = a.gates[(size_t)row * a.heads + head];
    } else {
      for (int r = tid; r < a.rank; r += nthr) a1[r] = mat_value<T, 1>(a.src, row, a.col_a() + r).v[0];
      __syncthreads();
    }
    const float decay = MEM ? expf(gate.x) : 0.f;
    for (int c = tid; c < dk; c += nthr) {
      const int ch = head * dk + c;
      q[c] = mat_value<T, 1>(a.src, row, a.col0 + ch).v[0] * a.q_scale;
      k[c] = mat_value<T, 1>(a.src, row, a.col_k() + ch).v[0];
      if constexpr (MEM) {
        k[c] *= gate.y;
        al[c] = decay;
        continue;
      }
      float z = a.a2_bias[ch];
      const float* w = a.a2 + (size_t)ch * a.rank;
      for (int r = 0; r < a.rank; ++r) z = fmaf(w[r], a1[r], z);
      al[c] = expf(log_sigmoid(z) * a.inv_tau);
    }
    __syncthreads();
    for (int c0 = ty < groups ? tx : dva; c0 * VEC < dva; c0 += a.cols) {
      const int c = c0 * VEC;
      Vec<VEC> v;
      if constexpr (MEM) v = memory_value<T, VEC>(a, row, head, c);
      else v = mat_value<T, VEC>(a.src, row, a.col_v() + head * dv + c);
      float acc[VEC] = {};
      constexpr int U = 8;
      for (int d0 = ty; d0 < dk; d0 += groups * U) {
        Vec<VEC> s[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int dd = d0 + u * groups;
          if (dd < dk && !fresh) s[u] = load_vec<VEC>(S + (size_t)dd * dvs + c);
          else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) s[u].v[e] = 0.f;
          }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int dd = d0 + u * groups;
          if (dd < dk) {
            const float aa = al[dd], kk = k[dd], qq = q[dd];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
              s[u].v[e] = fmaf(s[u].v[e], aa, kk * v.v[e]);
              acc[e] = fmaf(s[u].v[e], qq, acc[e]);
            }
            store_vec<VEC>(S + (size_t)dd * dvs + c, s[u]);
          }
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) red[ty * dvs + c + e] = acc[e];
    }
    __syncthreads();
    float ss = 0.f, inv = 1.f;
    if constexpr (MEM) {
      float qn = 0.f;
      for (int g = 0; g < groups; ++g) qn += red[g * dvs + dv];
      inv = 1.0f / (fmaxf(fabsf(qn), gate.z) + a.den_eps);
    }
    for (int c = tid; c < dv; c += nthr) {
      float o = red[c];
      for (int g = 1; g < groups; ++g) o += red[g * dvs + c];
      if constexpr (MEM) o *= inv;
      red[c] = o;  // (column c is read and written by this thread only)
      ss += o * o;
    }
    const float r = 1.0f / sqrtf(block_sum(ss, part) / (float)dv + a.eps);
    T* dst = (T*)a.out + (size_t)row * a.out_stride + (size_t)head * dv;
    for (int c = tid; c < dv; c += nthr) {
      const float g = mat_value<T, 1>(a.src, row, a.col_g + head * dv + c).v[0];
      if constexpr (MEM) st(dst + c, red[c] * r * a.norm[head * dv + c] * sigmoid(g) * a.out_scale);
      else st(dst + c, red[c] * r * a.norm[c] * silu(g));
    }
    __syncthreads();
  }
}

// ---- matrix memory: gates -----------------------------------------------------------------------------------------------
struct GateArgs {
  KvDev d;
  MemoryGates g;
  float* state;
  int rec_elems;
  const int *cu, *row_seq, *pos;
};

// One CTA per (request, head).  m_t = max(m_(t-1) + f_t, i_t) is a scan: the pair (F, M) stands for m -> max(m + F, M).
template <typename T>
__global__ void __launch_bounds__(1024) memory_gates_kernel(GateArgs a) {
  __shared__ float2 total[32];
  __shared__ float s_m[1025];
  const int req = blockIdx.x, head = blockIdx.y, H = a.g.heads, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
  const int r0 = a.cu[req], count = a.cu[req + 1] - r0;
  if (count <= 0 || a.d.state[ST_ERR] != 0) return;
  const int slot = a.row_seq[r0];
  if (slot < 0 || slot >= a.d.max_seqs) return;
  float* m_at = a.state + (size_t)slot * a.rec_elems + a.g.m_off + head;
  float m_in = a.pos[r0] == 0 ? 0.f : *m_at;
  auto capped = [&](int row, int col) {
    const float z = mat_value<T, 1>(a.g.src, row, col).v[0] + a.g.bias[col];
    return a.g.cap * tanhf(z / a.g.cap);
  };
  for (int base = 0; base < count; base += blockDim.x) {
    const int row = r0 + base + tid;
    const bool on = base + tid < count;
    float in = -INFINITY, forget = 0.f;
    if (on) {
      in = capped(row, head);
      forget = log_sigmoid(capped(row, H + head));
    }
    float F = forget, M = in;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) {
        M = fmaxf(Mp + F, M);
        F += Fp;
      }
    }
    if (lane == 31) total[warp] = make_float2(F, M);
    __syncthreads();
    float m_warp = m_in, m_end = m_in;
    for (int w = 0; w < n_warps; ++w) {
      if (w == warp) m_warp = m_end;
      m_end = fmaxf(m_end + total[w].x, total[w].y);
    }
    const float m = fmaxf(m_warp + F, M);
    if (tid == 0) s_m[0] = m_in;
    s_m[tid + 1] = m;
    __syncthreads();
    if (on) a.g.out[(size_t)row * H + head] = make_float4(forget + s_m[tid] - m, expf(in - m), expf(-m), 0.f);
    m_in = m_end;
    __syncthreads();
  }
  if (tid == 0) *m_at = m_in;
}

// ---- chunks: plan ------------------------------------------------------------------------------------------------
// One CTA: the chunks of every portion that goes chunk by chunk, and where each request's start.
__global__ void __launch_bounds__(1024) gla_plan_kernel(const int* __restrict__ cu, int n_req, int max_chunks, int4* __restrict__ plan,
                                                        int* __restrict__ first_chunk) {
  __shared__ int sums[32];
  __shared__ int base;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid == 0) base = 0;
  __syncthreads();
  for (int i0 = 0; i0 < n_req; i0 += blockDim.x) {
    const int i = i0 + tid;
    const int r0 = i < n_req ? cu[i] : 0, count = i < n_req ? cu[i + 1] - r0 : 0;
    const int n = count > kGlaStepTokens ? (count + kC - 1) / kC : 0;
    int inc = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int t = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += t;
    }
    if (lane == 31) sums[warp] = inc;
    __syncthreads();
    int before = base, total = 0;
    for (int w = 0; w < 32; ++w) {
      if (w < warp) before += sums[w];
      total += sums[w];
    }
    const int first = before + inc - n;
    if (i < n_req) {
      first_chunk[i] = first;
      for (int c = 0; c < n && first + c < max_chunks; ++c) plan[first + c] = make_int4(r0 + c * kC, min(kC, count - c * kC), i, 0);
    }
    __syncthreads();
    if (tid == 0) base += total;
    __syncthreads();
  }
  if (tid == 0) first_chunk[n_req] = min(base, max_chunks);
}

// ---- chunks: decays, scaled q and k, weights of the sum -------------------------------------------------------------
// The weights factor into (q_i e^{L_i - r}) . (k_j e^{r - L_j}) with r the sum at the start of i's half of the chunk: the first
// factor only shrinks, and the second only shrinks for keys of the other half.  Within a half it may grow, by at most e^kMaxGrowth
// on this route; a chunk whose decays are stronger takes the pairs one by one.
constexpr float kMaxGrowth = 60.f;

template <typename T, int VEC>
__global__ void __launch_bounds__(256) gla_chunk_kernel(Gla a) {
  extern __shared__ __align__(16) float sh[];
  __shared__ int s_range;
  const int chunk = blockIdx.x, head = blockIdx.y;
  if (chunk >= a.first_chunk[a.n_req] || a.d.state[ST_ERR] != 0) return;
  const int4 it = a.plan[chunk];
  const int dk = a.dk, dkp = a.dkp, ldr = dkp + 8, n = it.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *q = sh, *k = q + kC * ldr, *L = k + kC * ldr, *a1 = L + kC * ldr;
  unsigned char* out = a.chunks + ((size_t)chunk * a.heads + head) * a.chunk_bytes;
  if (tid == 0) s_range = 0;
  for (int i = tid; i < kC * a.rank; i += 256) {
    const int t = i / a.rank, r = i - t * a.rank;
    a1[i] = t < n ? mat_value<T, 1>(a.src, it.x + t, a.col_a() + r).v[0] : 0.f;
  }
  const int groups = dkp / VEC;
  for (int i = tid; i < kC * groups; i += 256) {
    const int t = i / groups, c = (i - t * groups) * VEC;
    Vec<VEC> x{}, y{};
    if (t < n && c < dk) {
      x = mat_value<T, VEC>(a.src, it.x + t, head * dk + c);
      y = mat_value<T, VEC>(a.src, it.x + t, a.col_k() + head * dk + c);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) x.v[e] *= a.q_scale;
    store_vec<VEC>(q + t * ldr + c, x);
    store_vec<VEC>(k + t * ldr + c, y);
  }
  __syncthreads();
  for (int i = tid; i < 4 * dkp; i += 256) {  // eight tokens of one key channel
    const int part = i / dkp, c = i - part * dkp, t0 = part * 8;
    float z[8];
    const float b = c < dk ? a.a2_bias[head * dk + c] : 0.f;
#pragma unroll
    for (int t = 0; t < 8; ++t) z[t] = b;
    if (c < dk) {
      const float* w = a.a2 + (size_t)(head * dk + c) * a.rank;
      for (int r = 0; r < a.rank; ++r) {
        const float wr = w[r];
#pragma unroll
        for (int t = 0; t < 8; ++t) z[t] = fmaf(wr, a1[(t0 + t) * a.rank + r], z[t]);
      }
    }
#pragma unroll
    for (int t = 0; t < 8; ++t) L[(t0 + t) * ldr + c] = c < dk && t0 + t < n ? log_sigmoid(z[t]) * a.inv_tau : 0.f;
  }
  __syncthreads();
  for (int c = tid; c < dkp; c += 256) {
    float s = 0.f, half = 0.f;
    for (int t = 0; t < kC; ++t) {
      if (t == 16) half = s;
      s += L[t * ldr + c];
      L[t * ldr + c] = s;
    }
    atomicMax(&s_range, __float_as_int(fmaxf(-half, half - s)));  // (both are >= 0: their bits order like the numbers)
    reinterpret_cast<float*>(out + off_decay(dkp))[c] = expf(s);
  }
  __syncthreads();
  for (int i = tid; i < kC * (dkp / 2); i += 256) {
    const int t = i / (dkp / 2), c = 2 * (i - t * (dkp / 2));
    const float2 lt = *reinterpret_cast<const float2*>(&L[t * ldr + c]), le = *reinterpret_cast<const float2*>(&L[(kC - 1) * ldr + c]);
    const float2 qt = *reinterpret_cast<const float2*>(&q[t * ldr + c]), kt = *reinterpret_cast<const float2*>(&k[t * ldr + c]);
    uint32_t hi, lo;
    split_bf16(qt.x * expf(lt.x), qt.y * expf(lt.y), hi, lo);
    unsigned char* at = out + (size_t)t * qk_row(dkp) + c * 2;
    *reinterpret_cast<uint32_t*>(at + off_part(dkp, 0)) = hi;
    *reinterpret_cast<uint32_t*>(at + off_part(dkp, 1)) = lo;
    split_bf16(kt.x * expf(le.x - lt.x), kt.y * expf(le.y - lt.y), hi, lo);
    *reinterpret_cast<uint32_t*>(at + off_part(dkp, 2)) = hi;
    *reinterpret_cast<uint32_t*>(at + off_part(dkp, 3)) = lo;
  }
  constexpr int kPer = kScanCols / VEC;
  for (int i = tid; i < a.n_slices * kC * kPer; i += 256) {
    const int s = i / (kC * kPer), rest = i - s * kC * kPer, t = rest / kPer, c = (rest - t * kPer) * VEC, col = s * kScanCols + c;
    Vec<VEC> v{};
    if (t < n && col < a.dv) v = mat_value<T, VEC>(a.src, it.x + t, a.col_v() + head * a.dv + col);
    unsigned char* dst = a.values + ((size_t)chunk * a.heads + head) * a.v_bytes + (size_t)s * kVSlice + (size_t)t * kVRow + c * 2;
    store_vec<VEC>(reinterpret_cast<__nv_bfloat16*>(dst), v);
  }
  unsigned char *ahi = out + off_a(dkp, 0), *alo = out + off_a(dkp, 1);
  if (__int_as_float(s_range) >= kMaxGrowth) {
    for (int i = warp; i < kC; i += 8) {
      const int j = lane;
      float s = 0.f;
      if (j <= i)
        for (int c = 0; c < dk; ++c) s = fmaf(q[i * ldr + c] * k[j * ldr + c], expf(L[i * ldr + c] - L[j * ldr + c]), s);
      const __nv_bfloat16 h = __float2bfloat16(s);
      *reinterpret_cast<__nv_bfloat16*>(ahi + i * kARow + j * 2) = h;
      *reinterpret_cast<__nv_bfloat16*>(alo + i * kARow + j * 2) = __float2bfloat16(s - __bfloat162float(h));
    }
    return;
  }
  // 16 x 8 tiles: warps 0, 1 the first half's keys of the first half, warps 2..5 all keys of the second half, 6, 7 the zeros
  const int g = lane >> 2, t = lane & 3, I = warp >= 2 && warp < 6 ? 1 : 0, nt = warp < 2 ? warp : (warp < 6 ? warp - 2 : warp - 4);
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  if (warp < 6) {
    const float* ref = I ? &L[15 * ldr] : nullptr;
    const int i0 = 16 * I + g, i1 = i0 + 8, j = 8 * nt + g;
    auto at2 = [&](const float* p) { return *reinterpret_cast<const float2*>(p); };
    for (int ks = 0; ks < dkp / 16; ++ks) {
      uint32_t qh[4], ql[4], kh[2], kl[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int c = ks * 16 + h * 8 + 2 * t;
        const float2 r = ref ? at2(ref + c) : make_float2(0.f, 0.f);
        const float2 l0 = at2(&L[i0 * ldr + c]), l1 = at2(&L[i1 * ldr + c]), lj = at2(&L[j * ldr + c]);
        const float2 q0 = at2(&q[i0 * ldr + c]), q1 = at2(&q[i1 * ldr + c]), kj = at2(&k[j * ldr + c]);
        split_bf16(q0.x * expf(l0.x - r.x), q0.y * expf(l0.y - r.y), qh[2 * h], ql[2 * h]);
        split_bf16(q1.x * expf(l1.x - r.x), q1.y * expf(l1.y - r.y), qh[2 * h + 1], ql[2 * h + 1]);
        split_bf16(kj.x * expf(r.x - lj.x), kj.y * expf(r.y - lj.y), kh[h], kl[h]);
      }
      mma16816(acc, qh, kh[0], kh[1]);
      mma16816(acc, qh, kl[0], kl[1]);
      mma16816(acc, ql, kh[0], kh[1]);
    }
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int i = 16 * I + g + 8 * h, j = 8 * nt + 2 * t;
    const float x = j <= i ? acc[2 * h] : 0.f, y = j + 1 <= i ? acc[2 * h + 1] : 0.f;
    uint32_t hi, lo;
    split_bf16(x, y, hi, lo);
    *reinterpret_cast<uint32_t*>(ahi + i * kARow + j * 2) = hi;
    *reinterpret_cast<uint32_t*>(alo + i * kARow + j * 2) = lo;
  }
}

// ---- chunks: the walk ------------------------------------------------------------------------------------------------
// One warp holds 16 value columns of S^T [dv][dk] as MMA accumulators, which are at the same time the A operand of
// o^T = S^T q^T.  A ring of stages, each a chunk's block and its slice of values (two bulk copies).
// DELTA: the values that enter the state are u = U - W S with the state at the chunk's start, W [tokens][dk] and U [tokens][dv] made by
// delta_chunk_kernel (delta.cu); u is f32 and enters the tensor cores as two terms.
template <int NT, bool DELTA>  // NT: 8-channel tiles of the state a warp holds
__global__ void __launch_bounds__(kScanWarps * 32) gla_scan_kernel(Gla a) {
  extern __shared__ unsigned char scan_dyn[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(scan_dyn) + 127) & ~(uintptr_t)127);
  const int req = blockIdx.x, head = blockIdx.y, slice = blockIdx.z;
  const int c0 = a.first_chunk[req], c1 = a.first_chunk[req + 1];
  if (c0 >= c1 || a.d.state[ST_ERR] != 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int dkp = a.dkp, n_t = dkp / 8, stages = a.stages;
  constexpr uint32_t vbytes = (uint32_t)(DELTA ? kUSlice : kVSlice);
  const uint32_t cbytes = (uint32_t)(DELTA ? delta_chunk_size(dkp) : chunk_size(dkp)), stage_bytes = cbytes + vbytes;
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + (size_t)stages * stage_bytes);
  const int r0 = a.cu[req], slot = a.row_seq[r0];
  if (slot < 0 || slot >= a.d.max_seqs) return;
  if (tid == 0) {
    for (int s = 0; s < stages; ++s) ptx::mbar_init(&full[s], 1);
    ptx::mbar_fence_init();
  }
  __syncthreads();
  auto load = [&](int c, int s) {
    unsigned char* dst = smem + (size_t)s * stage_bytes;
    const size_t ch = (size_t)c * a.heads + head;
    ptx::mbar_expect_tx(&full[s], stage_bytes);
    ptx::bulk_g2s(dst, a.chunks + ch * a.chunk_bytes, cbytes, &full[s]);
    ptx::bulk_g2s(dst + cbytes, a.values + ch * a.v_bytes + (size_t)slice * vbytes, vbytes, &full[s]);
  };
  if (tid == 0)
    for (int s = 0; s < stages && c0 + s < c1; ++s) load(c0 + s, s);

  const int m0 = slice * kScanCols + warp * 16;  // first value column of the warp
  float* S = a.state + (size_t)slot * a.rec_elems + (size_t)head * a.dk * a.dvs;
  float acc[NT][4];
  const bool fresh = a.pos[r0] == 0;
#pragma unroll
  for (int j = 0; j < NT; ++j) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int col = m0 + g + (e >> 1) * 8, ch = j * 8 + 2 * t + (e & 1);
      acc[j][e] = !fresh && ch < a.dk && col < a.dva ? S[(size_t)ch * a.dvs + col] : 0.f;
    }
  }
  bool ok = true;
  int s = 0;
  uint32_t ph = 0;
  for (int c = c0; c < c1; ++c) {
    ok = ptx::mbar_wait(&full[s], ph);
    if (!__syncthreads_and(ok)) break;
    const unsigned char* st_ = smem + (size_t)s * stage_bytes;
    const uint32_t base = ptx::smem_u32(st_), vbase = base + cbytes;
    const int lr = lane & 7, lm = lane >> 3;
    float o[4][4], w[4][4];  // w: W S
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
      w[n][0] = w[n][1] = w[n][2] = w[n][3] = 0.f;
    }
    // from the state: k = channels.  One ldmatrix.x4 covers 8 tokens x 32 channels (two k steps).
#pragma unroll
    for (int kk = 0; kk < NT / 4; ++kk) {
      if (kk * 4 < n_t) {
        uint32_t sh_[2][4], sl_[2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int j = kk * 4 + u * 2;
          split_bf16(acc[j][0], acc[j][1], sh_[u][0], sl_[u][0]);
          split_bf16(acc[j][2], acc[j][3], sh_[u][1], sl_[u][1]);
          split_bf16(acc[j + 1][0], acc[j + 1][1], sh_[u][2], sl_[u][2]);
          split_bf16(acc[j + 1][2], acc[j + 1][3], sh_[u][3], sl_[u][3]);
        }
        // two tiles of tokens side by side (and o beside w), so that an MMA does not wait for the one before it
#pragma unroll
        for (int n = 0; n < 4; n += 2) {
          uint32_t qh[2][4], ql[2][4], wh[2][4], wl[2][4];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const uint32_t at = base + (uint32_t)(((n + e) * 8 + lr) * qk_row(dkp) + kk * 64 + lm * 16);
            ldsm4(at + (uint32_t)off_part(dkp, 0), qh[e]);
            ldsm4(at + (uint32_t)off_part(dkp, 1), ql[e]);
            if constexpr (DELTA) {
              ldsm4(at + (uint32_t)off_w(dkp, 0), wh[e]);
              ldsm4(at + (uint32_t)off_w(dkp, 1), wl[e]);
            }
          }
#pragma unroll
          for (int u = 0; u < 2; ++u) {
#pragma unroll
            for (int term = 0; term < 3; ++term) {  // value x value, value x remainder, remainder x value
#pragma unroll
              for (int e = 0; e < 2; ++e) {
                const uint32_t* q = term == 1 ? ql[e] : qh[e];
                mma16816(o[n + e], term == 2 ? sl_[u] : sh_[u], q[2 * u], q[2 * u + 1]);
                if constexpr (DELTA) {
                  const uint32_t* x = term == 1 ? wl[e] : wh[e];
                  mma16816(w[n + e], term == 2 ? sl_[u] : sh_[u], x[2 * u], x[2 * u + 1]);
                }
              }
            }
          }
        }
      }
    }
    // v^T as A operand: rows = value columns, k = tokens (two steps of 16)
    uint32_t va[2][4], vr[2][4];  // vr: the remainders
    if constexpr (DELTA) {
      const float* U = reinterpret_cast<const float*>(st_ + cbytes) + (warp * 16 + g) * kUStride + 2 * t;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const float2 x = *reinterpret_cast<const float2*>(U + n * 8), y = *reinterpret_cast<const float2*>(U + 8 * kUStride + n * 8);
        split_bf16(x.x - w[n][0], x.y - w[n][1], va[n >> 1][(n & 1) * 2], vr[n >> 1][(n & 1) * 2]);
        split_bf16(y.x - w[n][2], y.y - w[n][3], va[n >> 1][(n & 1) * 2 + 1], vr[n >> 1][(n & 1) * 2 + 1]);
      }
    } else {
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        // the four 8 x 8 blocks of v [tokens][columns], transposed: (cols 0-7, tok 0-7), (cols 8-15, tok 0-7), (cols 0-7, tok 8-15), ...
        const int row = u * 16 + (lm >> 1) * 8 + lr, col = warp * 16 + (lm & 1) * 8;
        ldsm4_trans(vbase + (uint32_t)(row * kVRow + col * 2), va[u]);
      }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      uint32_t bh[4], bl[4];
      const uint32_t at = base + (uint32_t)((n * 8 + lr) * kARow + lm * 16);
      ldsm4(at + (uint32_t)off_a(dkp, 0), bh);
      ldsm4(at + (uint32_t)off_a(dkp, 1), bl);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        mma16816(o[n], va[u], bh[2 * u], bh[2 * u + 1]);
        mma16816(o[n], va[u], bl[2 * u], bl[2 * u + 1]);
        if constexpr (DELTA) mma16816(o[n], vr[u], bh[2 * u], bh[2 * u + 1]);
      }
    }
    // the state moves on: decay its columns, add v^T k
    const float* dec = reinterpret_cast<const float*>(st_ + off_decay(dkp));
#pragma unroll
    for (int j = 0; j < NT; j += 4) {
      if (j < n_t) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 d = *reinterpret_cast<const float2*>(dec + (j + e) * 8 + 2 * t);
          acc[j + e][0] *= d.x; acc[j + e][1] *= d.y; acc[j + e][2] *= d.x; acc[j + e][3] *= d.y;
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          uint32_t b[2][2][4];  // [value, remainder][pair of tiles]: k [tokens][channels], transposed: tokens 0-7 / 8-15 of the step x channels 0-7 / 8-15
#pragma unroll
          for (int p = 0; p < 2; ++p) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int row = u * 16 + (lm & 1) * 8 + lr, col = (j + 2 * e) * 8 + (lm >> 1) * 8;
              ldsm4_trans(base + (uint32_t)(off_part(dkp, 2 + p) + row * qk_row(dkp) + col * 2), b[p][e]);
            }
          }
#pragma unroll
          for (int term = 0; term < (DELTA ? 3 : 2); ++term) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const uint32_t* k = b[term == 1 ? 1 : 0][e >> 1] + 2 * (e & 1);
              mma16816(acc[j + e], term == 2 ? vr[u] : va[u], k[0], k[1]);
            }
          }
        }
      }
    }
    const int row0 = a.plan[c].x, rows = a.plan[c].y;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int tok = n * 8 + 2 * t + (e & 1), col = m0 + g + (e >> 1) * 8;
        if (tok < rows && col < a.dva) a.o[((size_t)(row0 + tok) * a.heads + head) * a.dvs + col] = o[n][e];
      }
    }
    __syncthreads();  // every warp has read the stage
    if (tid == 0 && c + stages < c1) {
      ptx::fence_proxy_async_smem();
      load(c + stages, s);
    }
    if (++s == stages) { s = 0; ph ^= 1u; }
  }
  if (!ok) { atomicExch(a.d.state + ST_ATTN_ERR, B200_ERR_DEVICE_FLAGGED); return; }
#pragma unroll
  for (int j = 0; j < NT; ++j) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int col = m0 + g + (e >> 1) * 8, ch = j * 8 + 2 * t + (e & 1);
      if (ch < a.dk && col < a.dva) S[(size_t)ch * a.dvs + col] = acc[j][e];
    }
  }
}

// ---- chunks: norm and gate -------------------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void __launch_bounds__(256) gla_out_kernel(Gla a) {
  const int chunk = blockIdx.x, head = blockIdx.y, lane = threadIdx.x & 31;
  if (chunk >= a.first_chunk[a.n_req] || a.d.state[ST_ERR] != 0) return;
  const int4 it = a.plan[chunk];
  for (int i = threadIdx.x >> 5; i < it.y; i += 8) {
    const int row = it.x + i;
    const float* o = a.o + ((size_t)row * a.heads + head) * a.dv;
    float ss = 0.f;
    for (int c = lane * VEC; c < a.dv; c += 32 * VEC) {
      const Vec<VEC> x = load_vec<VEC>(o + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += x.v[e] * x.v[e];
    }
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)a.dv + a.eps);
    T* dst = (T*)a.out + (size_t)row * a.out_stride + (size_t)head * a.dv;
    for (int c = lane * VEC; c < a.dv; c += 32 * VEC) {
      Vec<VEC> x = load_vec<VEC>(o + c);
      const Vec<VEC> w = load_vec<VEC>(a.norm + c), g = mat_value<T, VEC>(a.src, row, a.col_g + head * a.dv + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x.v[e] *= r * w.v[e] * g.v[e] * sigmoid_for<T>(g.v[e]);
      store_vec<VEC>(dst + c, x);
    }
  }
}

// ---- chunks of a matrix memory -----------------------------------------------------------------------------------------
// One decay for all channels: the weights are (q_i . k_j) e^(L_i - L_j) w_j, so the exponentials stay out of the product and decays of
// any strength take this route.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) memory_chunk_kernel(Gla a) {
  extern __shared__ __align__(16) float sh[];
  __shared__ float s_L[kC], s_w[kC];
  const int chunk = blockIdx.x, head = blockIdx.y;
  if (chunk >= a.first_chunk[a.n_req] || a.d.state[ST_ERR] != 0) return;
  const int4 it = a.plan[chunk];
  const int dk = a.dk, dkp = a.dkp, ldr = dkp + 8, n = it.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *q = sh, *k = q + kC * ldr;
  unsigned char* out = a.chunks + ((size_t)chunk * a.heads + head) * a.chunk_bytes;
  if (warp == 0) {
    float4 g{};
    if (lane < n) g = a.gates[(size_t)(it.x + lane) * a.heads + head];
    float L = g.x;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, L, o);
      if (lane >= o) L += x;
    }
    s_L[lane] = L;
    s_w[lane] = g.y;
  }
  const int groups = dkp / VEC;
  for (int i = tid; i < kC * groups; i += 256) {
    const int t = i / groups, c = (i - t * groups) * VEC;
    Vec<VEC> x{}, y{};
    if (t < n && c < dk) {
      x = mat_value<T, VEC>(a.src, it.x + t, a.col0 + head * dk + c);
      y = mat_value<T, VEC>(a.src, it.x + t, a.col_k() + head * dk + c);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) x.v[e] *= a.q_scale;
    store_vec<VEC>(q + t * ldr + c, x);
    store_vec<VEC>(k + t * ldr + c, y);
  }
  constexpr int kPer = kScanCols / VEC;
  for (int i = tid; i < a.n_slices * kC * kPer; i += 256) {
    const int s = i / (kC * kPer), rest = i - s * kC * kPer, t = rest / kPer, c = (rest - t * kPer) * VEC;
    Vec<VEC> v{};
    if (t < n) v = memory_value<T, VEC>(a, it.x + t, head, s * kScanCols + c);
    unsigned char* dst = a.values + ((size_t)chunk * a.heads + head) * a.v_bytes + (size_t)s * kVSlice + (size_t)t * kVRow + c * 2;
    store_vec<VEC>(reinterpret_cast<__nv_bfloat16*>(dst), v);
  }
  __syncthreads();
  const float end = s_L[kC - 1];
  for (int c = tid; c < dkp; c += 256) reinterpret_cast<float*>(out + off_decay(dkp))[c] = expf(end);
  for (int i = tid; i < kC * (dkp / 2); i += 256) {
    const int t = i / (dkp / 2), c = 2 * (i - t * (dkp / 2));
    const float fq = expf(s_L[t]), fk = s_w[t] * expf(end - s_L[t]);
    const float2 qt = *reinterpret_cast<const float2*>(&q[t * ldr + c]), kt = *reinterpret_cast<const float2*>(&k[t * ldr + c]);
    uint32_t hi, lo;
    split_bf16(qt.x * fq, qt.y * fq, hi, lo);
    unsigned char* at = out + (size_t)t * qk_row(dkp) + c * 2;
    *reinterpret_cast<uint32_t*>(at + off_part(dkp, 0)) = hi;
    *reinterpret_cast<uint32_t*>(at + off_part(dkp, 1)) = lo;
    split_bf16(kt.x * fk, kt.y * fk, hi, lo);
    *reinterpret_cast<uint32_t*>(at + off_part(dkp, 2)) = hi;
    *reinterpret_cast<uint32_t*>(at + off_part(dkp, 3)) = lo;
  }
  // 16 x 8 tiles, as in gla_chunk_kernel
  unsigned char *ahi = out + off_a(dkp, 0), *alo = out + off_a(dkp, 1);
  const int g = lane >> 2, t = lane & 3, I = warp >= 2 && warp < 6 ? 1 : 0, nt = warp < 2 ? warp : (warp < 6 ? warp - 2 : warp - 4);
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  if (warp < 6) {
    const int i0 = 16 * I + g, i1 = i0 + 8, j = 8 * nt + g;
    auto at2 = [&](const float* p) { return *reinterpret_cast<const float2*>(p); };
    for (int ks = 0; ks < dkp / 16; ++ks) {
      uint32_t qh[4], ql[4], kh[2], kl[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int c = ks * 16 + h * 8 + 2 * t;
        const float2 q0 = at2(&q[i0 * ldr + c]), q1 = at2(&q[i1 * ldr + c]), kj = at2(&k[j * ldr + c]);
        split_bf16(q0.x, q0.y, qh[2 * h], ql[2 * h]);
        split_bf16(q1.x, q1.y, qh[2 * h + 1], ql[2 * h + 1]);
        split_bf16(kj.x, kj.y, kh[h], kl[h]);
      }
      mma16816(acc, qh, kh[0], kh[1]);
      mma16816(acc, qh, kl[0], kl[1]);
      mma16816(acc, ql, kh[0], kh[1]);
    }
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int i = 16 * I + g + 8 * h, j = 8 * nt + 2 * t;
    const float x = j <= i ? acc[2 * h] * expf(s_L[i] - s_L[j]) * s_w[j] : 0.f;
    const float y = j + 1 <= i ? acc[2 * h + 1] * expf(s_L[i] - s_L[j + 1]) * s_w[j + 1] : 0.f;
    uint32_t hi, lo;
    split_bf16(x, y, hi, lo);
    *reinterpret_cast<uint32_t*>(ahi + i * kARow + j * 2) = hi;
    *reinterpret_cast<uint32_t*>(alo + i * kARow + j * 2) = lo;
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) memory_out_kernel(Gla a) {
  const int chunk = blockIdx.x, head = blockIdx.y, lane = threadIdx.x & 31;
  if (chunk >= a.first_chunk[a.n_req] || a.d.state[ST_ERR] != 0) return;
  const int4 it = a.plan[chunk];
  for (int i = threadIdx.x >> 5; i < it.y; i += 8) {
    const int row = it.x + i;
    const float* o = a.o + ((size_t)row * a.heads + head) * a.dvs;
    const float inv = 1.0f / (fmaxf(fabsf(o[a.dv]), a.gates[(size_t)row * a.heads + head].z) + a.den_eps);
    float ss = 0.f;
    for (int c = lane * VEC; c < a.dv; c += 32 * VEC) {
      const Vec<VEC> x = load_vec<VEC>(o + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += x.v[e] * inv * (x.v[e] * inv);
    }
    const float r = inv / sqrtf(warp_sum(ss) / (float)a.dv + a.eps) * a.out_scale;
    T* dst = (T*)a.out + (size_t)row * a.out_stride + (size_t)head * a.dv;
    for (int c = lane * VEC; c < a.dv; c += 32 * VEC) {
      Vec<VEC> x = load_vec<VEC>(o + c);
      const Vec<VEC> w = load_vec<VEC>(a.norm + head * a.dv + c), g = mat_value<T, VEC>(a.src, row, a.col_g + head * a.dv + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x.v[e] *= r * w.v[e] * sigmoid(g.v[e]);
      store_vec<VEC>(dst + c, x);
    }
  }
}

template <int NT, bool DELTA>
b200_status launch_scan(Gla& a, int n_req, cudaStream_t s) {
  const size_t stage = DELTA ? delta_chunk_size(a.dkp) + kUSlice : chunk_size(a.dkp) + kVSlice;
  a.stages = (int)std::min<size_t>(4, (220 * 1024) / stage);
  const size_t smem = a.stages * (stage + sizeof(uint64_t)) + 128;
  static bool configured = false;
  if (!configured) {
    B200_CUDA_TRY((cudaFuncSetAttribute(gla_scan_kernel<NT, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024)));
    configured = true;
  }
  gla_scan_kernel<NT, DELTA><<<dim3(n_req, a.heads, a.n_slices), kScanWarps * 32, smem, s>>>(a);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

template <bool DELTA>
b200_status launch_scan_of(Gla& a, int n_req, cudaStream_t s) {
  if (a.dkp <= 32) return launch_scan<4, DELTA>(a, n_req, s);
  if (a.dkp <= 64) return launch_scan<8, DELTA>(a, n_req, s);
  return a.dkp <= 128 ? launch_scan<16, DELTA>(a, n_req, s) : launch_scan<32, DELTA>(a, n_req, s);
}

}  // namespace

b200_status b200_gla_scan(Gla& a, int n_req, bool delta, cudaStream_t s) { return delta ? launch_scan_of<true>(a, n_req, s) : launch_scan_of<false>(a, n_req, s); }

b200_status b200_gla_out(const Gla& a, int chunks, bool wide, cudaStream_t s) {
  auto* kernel = wide ? gla_out_kernel<__nv_bfloat16, 4> : gla_out_kernel<__nv_bfloat16, 1>;
  kernel<<<dim3(chunks, a.heads), 256, 0, s>>>(a);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

bool b200_gla_takes_chunks(int dk, int dv, int elem_bytes) { return elem_bytes == 2 && dk <= 256; }

void GlaScratch::need(int heads, int dk, int dv, bool delta) {
  chunk_bytes = std::max(chunk_bytes, heads * (delta ? delta_chunk_size(pad_channels(dk)) : chunk_size(pad_channels(dk))));
  v_bytes = std::max(v_bytes, heads * slices_of(dv) * (delta ? kUSlice : kVSlice));
  o_elems = std::max(o_elems, (size_t)heads * dv);
}

void GlaScratch::need_delta(int heads, int kv_heads, int dk, int dv, bool chunks) {
  if (chunks) need(heads, dk, dv, true);
  row_elems = std::max(row_elems, ((size_t)2 * kv_heads * dk + (size_t)heads * dv + 3) / 4 * 4);
  gate_heads = std::max(gate_heads, heads);
}

bool GlaScratch::alloc() {
  max_chunks = max_rows / kC + max_reqs;
  auto get = [](auto** p, size_t bytes) { return cudaMalloc((void**)p, std::max<size_t>(bytes, 16)) == cudaSuccess; };
  return get(&chunks, max_chunks * chunk_bytes) && get(&values, max_chunks * v_bytes) && get(&o, sizeof(float) * o_elems * max_rows) &&
         get(&plan, sizeof(int4) * max_chunks) && get(&first_chunk, sizeof(int) * (max_reqs + 1)) &&
         get(&rows, sizeof(float) * row_elems * max_rows) && get(&gates, sizeof(float2) * gate_heads * max_rows);
}

void GlaScratch::free() {
  void* ptrs[] = {chunks, values, o, plan, first_chunk, rows, gates};
  for (void* p : ptrs) if (p) cudaFree(p);
}

b200_status b200_gla_plan(GlaScratch& g, const int32_t* d_cu, int n_req, int total_rows, void* stream) {
  if (n_req > g.max_reqs || total_rows > g.max_rows) { b200_set_error("gla: %d requests / %d rows exceed the scratch", n_req, total_rows); return B200_ERR_CAPACITY; }
  gla_plan_kernel<<<1, 1024, 0, (cudaStream_t)stream>>>(d_cu, n_req, g.max_chunks, g.plan, g.first_chunk);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

b200_status b200_memory_gates(b200_kv* kv, const MemoryGates& g, const int32_t* d_cu, const int32_t* d_row_seq, const int32_t* d_pos, int n_req,
                              int total_rows, void* stream) {
  if (g.layer < 0 || g.layer >= kv->cfg.n_layers || kv->lay[g.layer].rec_elems < g.m_off + g.heads) {
    b200_set_error("matrix memory: layer %d of the pool has no room for %d maxima", g.layer, g.heads);
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (n_req <= 0 || total_rows <= 0) return B200_OK;
  GateArgs a;
  a.d = kv->dev; a.g = g; a.state = kv->dev.rec_pool + kv->lay[g.layer].rec_off; a.rec_elems = kv->lay[g.layer].rec_elems;
  a.cu = d_cu; a.row_seq = d_row_seq; a.pos = d_pos;
  auto* kernel = kv->dev.elem_bytes == 4 ? memory_gates_kernel<float> : memory_gates_kernel<__nv_bfloat16>;
  kernel<<<dim3(n_req, g.heads), total_rows > 256 * n_req ? 1024 : (total_rows > 4 * n_req ? 256 : 32), 0, (cudaStream_t)stream>>>(a);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

b200_status b200_gla_run(b200_kv* kv, const GlaScratch& g, const GlaCall& c, const int32_t* d_cu, const int32_t* d_row_seq,
                         const int32_t* d_pos, int n_req, int total_rows, bool chunked, void* stream) {
  const bool mem = c.gates != nullptr;
  if (c.layer < 0 || c.layer >= kv->cfg.n_layers ||
      (mem ? kv->lay[c.layer].rec_elems < b200_memory_elems(c.heads, c.dk, c.dv) : kv->lay[c.layer].rec_elems < c.heads * c.dk * c.dv)) {
    b200_set_error("gla: layer %d of the pool has no state of %d x %d x %d", c.layer, c.heads, c.dk, c.dv);
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (n_req <= 0 || total_rows <= 0) return B200_OK;
  const bool f32 = kv->dev.elem_bytes == 4;
  cudaStream_t s = (cudaStream_t)stream;
  Gla a;
  a.d = kv->dev;
  a.state = kv->dev.rec_pool + kv->lay[c.layer].rec_off;
  a.rec_elems = kv->lay[c.layer].rec_elems;
  a.heads = c.heads; a.dk = c.dk; a.dv = c.dv; a.rank = c.rank; a.dkp = pad_channels(c.dk);
  a.dva = mem ? c.dv + 1 : c.dv; a.dvs = mem ? b200_memory_width(c.dv) : c.dv;
  a.col_g = c.col0 + 2 * c.heads * c.dk + c.heads * c.dv;
  a.gates = c.gates; a.col0 = c.col0; a.den_eps = c.den_eps; a.out_scale = c.out_scale;
  a.src = c.src; a.a2 = c.a2; a.a2_bias = c.a2_bias; a.norm = c.norm; a.q_scale = c.q_scale; a.inv_tau = c.inv_tau; a.eps = c.eps;
  a.out = c.out; a.out_stride = c.out_stride; a.cu = d_cu; a.row_seq = d_row_seq; a.pos = d_pos; a.n_req = n_req; a.total_rows = total_rows;
  a.chunks = g.chunks; a.values = g.values; a.o = g.o; a.plan = g.plan; a.first_chunk = g.first_chunk;
  a.chunk_bytes = chunk_size(a.dkp);
  a.n_slices = slices_of(a.dva);
  a.v_bytes = a.n_slices * kVSlice;
  a.stages = 0;
  // portions that are longer than the step kernel's limit exist only if some request has more than one row
  a.chunked = chunked && b200_gla_takes_chunks(c.dk, c.dv, kv->dev.elem_bytes);
  const bool v4 = c.dk % 4 == 0 && c.dv % 4 == 0 && c.col0 % 4 == 0 && (c.src.ws || c.src.y_stride % 4 == 0);
  {
    a.cols = std::min(v4 ? a.dvs / 4 : a.dva, 256);
    a.groups = std::max(1, std::min(256 / a.cols, (c.dk + 7) / 8));
    const size_t smem = sizeof(float) * (3 * (size_t)c.dk + (mem ? 0 : c.rank) + (size_t)a.groups * a.dvs);
    if (smem > 200 * 1024) { b200_set_error("gla: head widths %d / %d are too large", c.dk, c.dv); return B200_ERR_UNSUPPORTED; }
    auto* kernel = f32 ? (v4 ? gla_step_kernel<float, 4, false> : gla_step_kernel<float, 1, false>)
                       : (v4 ? gla_step_kernel<__nv_bfloat16, 4, false> : gla_step_kernel<__nv_bfloat16, 1, false>);
    if (mem) kernel = f32 ? (v4 ? gla_step_kernel<float, 4, true> : gla_step_kernel<float, 1, true>)
                          : (v4 ? gla_step_kernel<__nv_bfloat16, 4, true> : gla_step_kernel<__nv_bfloat16, 1, true>);
    if (smem > 48 * 1024) B200_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kernel<<<dim3(n_req, c.heads), (a.cols * a.groups + 31) / 32 * 32, smem, s>>>(a);
    B200_LAUNCH_CHECK();
  }
  if (!a.chunked || total_rows <= n_req) return B200_OK;
  const int chunks = std::min(total_rows / kC + n_req, g.max_chunks);
  const size_t smem = sizeof(float) * ((mem ? 2 : 3) * (size_t)kC * (a.dkp + 8) + (mem ? 0 : (size_t)kC * c.rank));
  if (smem > 220 * 1024) { b200_set_error("gla: a decay projection of inner width %d is too large", c.rank); return B200_ERR_UNSUPPORTED; }
  static bool configured = false;
  if (!configured) {
    B200_CUDA_TRY((cudaFuncSetAttribute(gla_chunk_kernel<__nv_bfloat16, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024)));
    B200_CUDA_TRY((cudaFuncSetAttribute(gla_chunk_kernel<__nv_bfloat16, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024)));
    B200_CUDA_TRY((cudaFuncSetAttribute(memory_chunk_kernel<__nv_bfloat16, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024)));
    B200_CUDA_TRY((cudaFuncSetAttribute(memory_chunk_kernel<__nv_bfloat16, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024)));
    configured = true;
  }
  const bool wide = v4 && c.out_stride % 4 == 0;
  auto* chunk_kernel = mem ? (wide ? memory_chunk_kernel<__nv_bfloat16, 4> : memory_chunk_kernel<__nv_bfloat16, 1>)
                           : (wide ? gla_chunk_kernel<__nv_bfloat16, 4> : gla_chunk_kernel<__nv_bfloat16, 1>);
  chunk_kernel<<<dim3(chunks, c.heads), 256, smem, s>>>(a);
  B200_LAUNCH_CHECK();
  b200_status st = b200_gla_scan(a, n_req, false, s);
  if (st != B200_OK) return st;
  if (!mem) return b200_gla_out(a, chunks, wide, s);
  auto* out_kernel = wide ? memory_out_kernel<__nv_bfloat16, 4> : memory_out_kernel<__nv_bfloat16, 1>;
  out_kernel<<<dim3(chunks, c.heads), 256, 0, s>>>(a);
  B200_LAUNCH_CHECK();
  return B200_OK;
}
