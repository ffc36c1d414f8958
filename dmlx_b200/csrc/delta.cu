// Gated delta rule: per head a state S [dk][dv] in f32 that keeps values under keys.  A token lets S decay, reads what S holds under its key,
// and writes the difference to its own value back: S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q.  The state lives in the pool's
// slot of the sequence; a sequence at position 0 starts from zero, so slots need no clearing.
//
// delta_prep_kernel: behind the projection: convolutions and silu, unit vectors, decay and beta, all f32 from here on.
// delta_step_kernel: token by token, one CTA per (request, head) (decode, short portions, f32).  One pass over the state gives S^T k and
// S^T q; with them u and o = g S^T q + (k . q) u are known before the state moves on.  The state stays in registers where it fits.
//
// Longer portions go in chunks of 32 tokens.  With L_t the sum of log decays since the chunk's start and S_0 the state there, the u of
// a chunk solve (I + A) u = diag(beta) (V - diag(e^L) K S_0), A_tj = beta_t e^(L_t - L_j) (k_t . k_j) for j < t.  With T = (I + A)^(-1),
//   u = U - W S_0,  U = T diag(beta) V,  W = T diag(beta e^L) K,
//   o_t = S_0^T (q_t e^(L_t)) + sum_(j <= t) e^(L_t - L_j) (q_t . k_j) u_j,   S_C = e^(L_C) S_0 + sum_j (k_j e^(L_C - L_j)) u_j^T.
//   delta_chunk_kernel (chunk, head), all in parallel: T, W, U, the weights of o and the scaled q and k;
//   gla_scan_kernel    (gla.cu) walks the chunks with S^T in registers;
//   gla_out_kernel     norm and gate of the rows.
// Every exponent is at most 0.  f32 factors enter the tensor cores as two bf16 terms.
#include <cuda_bf16.h>

#include <algorithm>
#include <cmath>

#include "common.h"
#include "delta.cuh"
#include "gla_chunks.cuh"

namespace {

__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ---- in front of the recurrence ------------------------------------------------------------------------------------
struct PrepArgs {
  DeltaCall c;
  const int *pool_state, *cu, *row_to_req, *row_seq, *pos;
  int max_seqs, v_units;
  float* rows;    // [row][stride]: q | k | v
  int stride;
  float2* gates;  // [row][heads]: log decay, beta
  float q_scale;
};

// One warp per (R rows, unit): a head of q or k, 32 * VEC columns of v, or the gates of a row.
template <typename T, int VEC, int TAPS, int R>
__global__ void __launch_bounds__(256) delta_prep_kernel(PrepArgs a, int n_rows) {
  const DeltaCall& c = a.c;
  const int begin = blockIdx.x * R, end = min(begin + R, n_rows), lane = threadIdx.x & 31, unit = blockIdx.y * 8 + (threadIdx.x >> 5);
  const int heads_qk = 2 * c.kv_heads, KD = c.kv_heads * c.dk, VD = c.heads * c.dv;
  if (unit > heads_qk + a.v_units || a.pool_state[ST_ERR] != 0) return;
  if (unit == heads_qk + a.v_units) {
    const int col = 2 * KD + 2 * VD;
    for (int row = begin; row < end; ++row)
      for (int h = lane; h < c.heads; h += 32) {
        const float b = mat_value<T, 1>(c.src, row, col + h).v[0], z = mat_value<T, 1>(c.src, row, col + c.heads + h).v[0] + c.dt_bias[h];
        a.gates[(size_t)row * c.heads + h] = make_float2(-c.rate[h] * softplus(z), sigmoid(b));
      }
    return;
  }
  const bool is_v = unit >= heads_qk;
  const int n0 = is_v ? 2 * KD + (unit - heads_qk) * 32 * VEC : unit * c.dk, width = is_v ? min(32 * VEC, 2 * KD + VD - n0) : c.dk;
  const bool once = width <= 32 * VEC;  // a lane holds all it works on
  const float scale = unit < c.kv_heads ? a.q_scale : 1.f;
  auto value = [&](int row, int col) { return mat_value<T, VEC>(c.src, row, col); };
  auto activate = [&](Vec<VEC>& x, float& ss) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      x.v[e] *= sigmoid_for<T>(x.v[e]);
      ss += x.v[e] * x.v[e];
    }
  };
  auto at = [&](int row, int col) { return a.rows + (size_t)row * a.stride + n0 + col; };
  // unit length, and the store; wider heads than a lane holds are stored first and read again
  auto finish = [&](int row, Vec<VEC> x, float ss) {
    const float r = is_v ? 1.f : scale / sqrtf(warp_sum(ss) + kDeltaUnitEps);
    for (int col = lane * VEC; col < width; col += 32 * VEC) {
      if (!once) x = load_vec<VEC>(at(row, col));
#pragma unroll
      for (int e = 0; e < VEC; ++e) x.v[e] *= r;
      store_vec<VEC>(at(row, col), x);
    }
  };
  if constexpr (R > 1 && TAPS > 0) {
    if (begin + R <= n_rows && a.row_to_req[begin] == a.row_to_req[begin + R - 1] && begin - a.cu[a.row_to_req[begin]] >= TAPS - 1) {
      Vec<VEC> x[R];
      float ss[R] = {};
      for (int col = lane * VEC; col < width; col += 32 * VEC) {
        if (c.src.ws) {
          conv_values_inside<TAPS, R, VEC>(c.conv, value, begin, n0 + col, x);
        } else {  // rows the matmul wrote itself
          const T* y = (const T*)c.src.y + (size_t)begin * c.src.y_stride;
          conv_values_inside<TAPS, R, VEC>(c.conv, [&](int row, int k) { return load_vec<VEC>(y + (row - begin) * c.src.y_stride + k); }, begin, n0 + col, x);
        }
#pragma unroll
        for (int r = 0; r < R; ++r) {
          activate(x[r], ss[r]);
          if (!once) store_vec<VEC>(at(begin + r, col), x[r]);
        }
      }
#pragma unroll
      for (int r = 0; r < R; ++r) finish(begin + r, x[r], ss[r]);
      return;
    }
  }
  for (int first = begin; first < end; ++first) {
    const int req = a.row_to_req[first], r0 = a.cu[req], count = a.cu[req + 1] - r0, slot = a.row_seq[first];
    if (slot < 0 || slot >= a.max_seqs) continue;
    const int n = conv_rows(c.conv, first - r0, count);
    for (int row = first; row < first + n; ++row) {
      Vec<VEC> x{};
      float ss = 0.f;
      for (int col = lane * VEC; col < width; col += 32 * VEC) {
        x = conv_value<VEC>(c.conv, value, row, row - r0, a.pos[row], slot, n0 + col);
        activate(x, ss);
        if (!once) store_vec<VEC>(at(row, col), x);
      }
      finish(row, x, ss);
    }
    if (first == r0)
      for (int col = lane * VEC; col < width; col += 32 * VEC) conv_update<VEC>(c.conv, value, r0, count, slot, n0 + col);
  }
}

// ---- token by token ------------------------------------------------------------------------------------------------
struct Delta {
  Gla g;
  int kv_heads, stride;
  const float* rows;
  const float2* gates;
  __device__ const float* q(int row, int head) const { return rows + (size_t)row * stride + (head / (g.heads / kv_heads)) * g.dk; }
  __device__ const float* k(int row, int head) const { return q(row, head) + kv_heads * g.dk; }
  __device__ const float* v(int row, int head) const { return rows + (size_t)row * stride + 2 * kv_heads * g.dk + head * g.dv; }
};

// KEEP > 0: a thread keeps its KEEP rows x VEC columns of the state in registers over the tokens of a portion; 0: any size, the state
// stays in memory.
template <typename T, int VEC, int KEEP>
__global__ void __launch_bounds__(256, KEEP == 32 ? 1 : 2) delta_step_kernel(Delta a) {
  extern __shared__ float sh[];
  __shared__ float part[32];
  const int req = blockIdx.x, head = blockIdx.y, dk = a.g.dk, dv = a.g.dv;
  const int r0 = a.g.cu[req], count = a.g.cu[req + 1] - r0;
  if (count <= 0 || (a.g.chunked && count > kGlaStepTokens) || a.g.d.state[ST_ERR] != 0) return;
  const int groups = a.g.groups, cols = a.g.cols;
  float *red_k = sh, *red_q = red_k + groups * cols * VEC, *q = red_q + groups * cols * VEC, *k = q + dk, *out = k + dk;  // out [dv]
  const int tid = threadIdx.x, nthr = blockDim.x, lane = tid & 31, tx = tid % cols, ty = tid / cols;
  const bool on = ty < groups;
  const int slot = a.g.row_seq[r0];
  if (slot < 0 || slot >= a.g.d.max_seqs) return;
  float* S = a.g.state + (size_t)slot * a.g.rec_elems + (size_t)head * dk * dv;
  const bool fresh = a.g.pos[r0] == 0;
  Vec<VEC> s[KEEP > 0 ? KEEP : 1];
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int d = ty + i * groups;
      s[i] = Vec<VEC>{};
      if (on && d < dk && tx * VEC < dv && !fresh) s[i] = load_vec<VEC>(S + (size_t)d * dv + tx * VEC);
    }
  }
  for (int t = 0; t < count; ++t) {
    const int row = r0 + t;
    const float *qg = a.q(row, head), *kg = a.k(row, head), *vg = a.v(row, head);
    for (int c = tid; c < dk; c += nthr) {
      q[c] = qg[c];
      k[c] = kg[c];
    }
    const float2 gate = a.gates[(size_t)row * a.g.heads + head];
    const float decay = expf(gate.x), beta = gate.y;
    __syncthreads();
    float qk = 0.f;
    for (int c = lane; c < dk; c += 32) qk = fmaf(q[c], k[c], qk);
    qk = warp_sum(qk);
    for (int c0 = 0; c0 < dv; c0 += cols * VEC) {
      const int c = c0 + tx * VEC;
      const bool mine = on && c < dv;
      float hk[VEC] = {}, hq[VEC] = {};
      if (mine) {
        if constexpr (KEEP > 0) {
#pragma unroll
          for (int i = 0; i < KEEP; ++i) {
            const int d = ty + i * groups;
            if (d < dk) {
              const float kk = k[d], qq = q[d];
#pragma unroll
              for (int e = 0; e < VEC; ++e) {
                hk[e] = fmaf(s[i].v[e], kk, hk[e]);
                hq[e] = fmaf(s[i].v[e], qq, hq[e]);
              }
            }
          }
        } else if (!fresh || t > 0) {
#pragma unroll 8
          for (int d = ty; d < dk; d += groups) {
            const Vec<VEC> x = load_vec<VEC>(S + (size_t)d * dv + c);
            const float kk = k[d], qq = q[d];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
              hk[e] = fmaf(x.v[e], kk, hk[e]);
              hq[e] = fmaf(x.v[e], qq, hq[e]);
            }
          }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          red_k[ty * cols * VEC + tx * VEC + e] = hk[e];
          red_q[ty * cols * VEC + tx * VEC + e] = hq[e];
        }
      }
      __syncthreads();
      if (mine) {
        Vec<VEC> u = load_vec<VEC>(vg + c), held{}, read{};
        for (int g = 0; g < groups; ++g) {
          const Vec<VEC> x = load_vec<VEC>(red_k + g * cols * VEC + tx * VEC), y = load_vec<VEC>(red_q + g * cols * VEC + tx * VEC);
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            held.v[e] += x.v[e];
            read.v[e] += y.v[e];
          }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          u.v[e] = beta * (u.v[e] - decay * held.v[e]);
          if (ty == 0) out[c + e] = fmaf(decay, read.v[e], qk * u.v[e]);
        }
        if constexpr (KEEP > 0) {
#pragma unroll
          for (int i = 0; i < KEEP; ++i) {
            const int d = ty + i * groups;
            const float kk = d < dk ? k[d] : 0.f;
#pragma unroll
            for (int e = 0; e < VEC; ++e) s[i].v[e] = fmaf(decay, s[i].v[e], kk * u.v[e]);
          }
        } else {
#pragma unroll 8
          for (int d = ty; d < dk; d += groups) {
            Vec<VEC> x{};
            if (!fresh || t > 0) x = load_vec<VEC>(S + (size_t)d * dv + c);
            const float kk = k[d];
#pragma unroll
            for (int e = 0; e < VEC; ++e) x.v[e] = fmaf(decay, x.v[e], kk * u.v[e]);
            store_vec<VEC>(S + (size_t)d * dv + c, x);
          }
        }
      }
      __syncthreads();
    }
    float ss = 0.f;
    for (int c = tid; c < dv; c += nthr) ss += out[c] * out[c];
    const float r = 1.0f / sqrtf(block_sum(ss, part) / (float)dv + a.g.eps);
    T* dst = (T*)a.g.out + (size_t)row * a.g.out_stride + (size_t)head * dv;
    for (int c = tid; c < dv; c += nthr)
      st(dst + c, out[c] * r * a.g.norm[c] * silu(mat_value<T, 1>(a.g.src, row, a.g.col_g + head * dv + c).v[0]));
    __syncthreads();
  }
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int d = ty + i * groups;
      if (on && d < dk && tx * VEC < dv) store_vec<VEC>(S + (size_t)d * dv + tx * VEC, s[i]);
    }
  }
}

// ---- chunks ----------------------------------------------------------------------------------------------------------
constexpr int kLdT = kC + 2;  // the two halves of a broadcast lie in different banks

// 16 x 16 x 16 product of one (row, column) per thread.
__device__ __forceinline__ float dot16(const float* x, int dx, const float* y, int dy) {
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 16; ++i) s = fmaf(x[i * dx], y[i * dy], s);
  return s;
}

__global__ void __launch_bounds__(256, 3) delta_chunk_kernel(Delta a) {
  extern __shared__ __align__(16) float sh[];
  __shared__ float s_L[kC], s_beta[kC];
  const int chunk = blockIdx.x, head = blockIdx.y;
  if (chunk >= a.g.first_chunk[a.g.n_req] || a.g.d.state[ST_ERR] != 0) return;
  const int4 it = a.g.plan[chunk];
  const int dk = a.g.dk, dv = a.g.dv, dkp = a.g.dkp, ldr = dkp + 8, n = it.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *q = sh, *k = q + kC * ldr, *A = k + kC * ldr, *Ti = A + kC * kLdT;
  unsigned char* out = a.g.chunks + ((size_t)chunk * a.g.heads + head) * a.g.chunk_bytes;
  if (warp == 0) {
    float2 gate = make_float2(0.f, 0.f);
    if (lane < n) gate = a.gates[(size_t)(it.x + lane) * a.g.heads + head];
    float L = gate.x;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, L, o);
      if (lane >= o) L += x;
    }
    s_L[lane] = L;
    s_beta[lane] = gate.y;
  }
  const bool v4 = dk % 4 == 0;
#pragma unroll
  for (int t = warp; t < kC; t += 8) {
    const float *qg = a.q(it.x + min(t, n - 1), head), *kg = a.k(it.x + min(t, n - 1), head);
    if (v4) {
      for (int c = lane * 4; c < dkp; c += 128) {
        Vec<4> x{}, y{};
        if (t < n && c < dk) {
          x = load_vec<4>(qg + c);
          y = load_vec<4>(kg + c);
        }
        store_vec<4>(q + t * ldr + c, x);
        store_vec<4>(k + t * ldr + c, y);
      }
    } else {
      for (int c = lane; c < dkp; c += 32) {
        const bool in = t < n && c < dk;
        q[t * ldr + c] = in ? qg[c] : 0.f;
        k[t * ldr + c] = in ? kg[c] : 0.f;
      }
    }
  }
  __syncthreads();
  // q k^T and k k^T in 16 x 8 tiles: warps 0, 1 the first half's keys of the first half, warps 2..5 all keys of the second half
  const int g = lane >> 2, t = lane & 3;
  {
    unsigned char *mhi = out + off_a(dkp, 0), *mlo = out + off_a(dkp, 1);
    const int I = warp >= 2 && warp < 6 ? 1 : 0, nt = warp < 2 ? warp : (warp < 6 ? warp - 2 : warp - 4);
    float acc[4] = {0.f, 0.f, 0.f, 0.f}, kk[4] = {0.f, 0.f, 0.f, 0.f};
    if (warp < 6) {
      const int i0 = 16 * I + g, i1 = i0 + 8, j = 8 * nt + g;
      auto at2 = [&](const float* p) { return *reinterpret_cast<const float2*>(p); };
      for (int ks = 0; ks < dkp / 16; ++ks) {
        uint32_t qh[4], ql[4], xh[4], xl[4], kh[2], kl[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int c = ks * 16 + h * 8 + 2 * t;
          const float2 q0 = at2(&q[i0 * ldr + c]), q1 = at2(&q[i1 * ldr + c]), x0 = at2(&k[i0 * ldr + c]), x1 = at2(&k[i1 * ldr + c]), kj = at2(&k[j * ldr + c]);
          split_bf16(q0.x, q0.y, qh[2 * h], ql[2 * h]);
          split_bf16(q1.x, q1.y, qh[2 * h + 1], ql[2 * h + 1]);
          split_bf16(x0.x, x0.y, xh[2 * h], xl[2 * h]);
          split_bf16(x1.x, x1.y, xh[2 * h + 1], xl[2 * h + 1]);
          split_bf16(kj.x, kj.y, kh[h], kl[h]);
        }
        mma16816(acc, qh, kh[0], kh[1]);
        mma16816(acc, qh, kl[0], kl[1]);
        mma16816(acc, ql, kh[0], kh[1]);
        mma16816(kk, xh, kh[0], kh[1]);
        mma16816(kk, xh, kl[0], kl[1]);
        mma16816(kk, xl, kh[0], kh[1]);
      }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int i = 16 * I + g + 8 * h, j = 8 * nt + 2 * t;
      const float e0 = j <= i ? expf(s_L[i] - s_L[j]) : 0.f, e1 = j + 1 <= i ? expf(s_L[i] - s_L[j + 1]) : 0.f;
      uint32_t hi, lo;
      split_bf16(acc[2 * h] * e0, acc[2 * h + 1] * e1, hi, lo);
      *reinterpret_cast<uint32_t*>(mhi + i * kARow + j * 2) = hi;
      *reinterpret_cast<uint32_t*>(mlo + i * kARow + j * 2) = lo;
      *reinterpret_cast<float2*>(&A[i * kLdT + j]) = make_float2(j < i ? s_beta[i] * kk[2 * h] * e0 : 0.f, j + 1 < i ? s_beta[i] * kk[2 * h + 1] * e1 : 0.f);
    }
  }
  __syncthreads();
  const float end = s_L[kC - 1];
  if (warp == 0) {
    // the two diagonal blocks of T, a column per lane
    const int b0 = lane & 16, c = lane & 15;
    float x[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      float v = r == c ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < r; ++j) v = fmaf(-A[(b0 + r) * kLdT + b0 + j], x[j], v);
      x[r] = v;
    }
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      Ti[(b0 + r) * kLdT + b0 + c] = x[r];
      if (b0) Ti[r * kLdT + 16 + c] = 0.f;
    }
  } else {
    for (int c = tid - 32; c < dkp; c += 224) reinterpret_cast<float*>(out + off_decay(dkp))[c] = expf(end);
    for (int tok = warp - 1; tok < kC; tok += 7) {
      const float fq = expf(s_L[tok]), fk = expf(end - s_L[tok]);
      for (int c = lane * 4; c < dkp; c += 128) {
        const Vec<4> qt = load_vec<4>(&q[tok * ldr + c]), kt = load_vec<4>(&k[tok * ldr + c]);
        uint2 hi, lo;
        unsigned char* at = out + (size_t)tok * qk_row(dkp) + c * 2;
        split_bf16(qt.v[0] * fq, qt.v[1] * fq, hi.x, lo.x);
        split_bf16(qt.v[2] * fq, qt.v[3] * fq, hi.y, lo.y);
        *reinterpret_cast<uint2*>(at + off_part(dkp, 0)) = hi;
        *reinterpret_cast<uint2*>(at + off_part(dkp, 1)) = lo;
        split_bf16(kt.v[0] * fk, kt.v[1] * fk, hi.x, lo.x);
        split_bf16(kt.v[2] * fk, kt.v[3] * fk, hi.y, lo.y);
        *reinterpret_cast<uint2*>(at + off_part(dkp, 2)) = hi;
        *reinterpret_cast<uint2*>(at + off_part(dkp, 3)) = lo;
      }
    }
  }
  __syncthreads();
  {  // the block below the diagonal: - T_22 A_21 T_11, through the free upper right block of A
    const int r = tid >> 4, c = tid & 15;
    A[r * kLdT + 16 + c] = dot16(&A[(16 + r) * kLdT], 1, &Ti[c], kLdT);
    __syncthreads();
    Ti[(16 + r) * kLdT + c] = -dot16(&Ti[(16 + r) * kLdT + 16], 1, &A[16 + c], kLdT);
  }
  __syncthreads();
  // W = T diag(beta e^L) K: the blocks (0, 0), (1, 0) and (1, 1) of the weights as A operands
  {
    uint32_t th[3][4], tl[3][4];
#pragma unroll
    for (int b = 0; b < 3; ++b) {
      const int i = (b > 0 ? 16 : 0) + g, j0 = (b == 2 ? 16 : 0) + 2 * t;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int j = j0 + 8 * h;
        const float f0 = s_beta[j] * expf(s_L[j]), f1 = s_beta[j + 1] * expf(s_L[j + 1]);
        split_bf16(Ti[i * kLdT + j] * f0, Ti[i * kLdT + j + 1] * f1, th[b][2 * h], tl[b][2 * h]);
        split_bf16(Ti[(i + 8) * kLdT + j] * f0, Ti[(i + 8) * kLdT + j + 1] * f1, th[b][2 * h + 1], tl[b][2 * h + 1]);
      }
    }
    for (int nt = warp; nt < dkp / 8; nt += 8) {
      uint32_t kh[2][2], kl[2][2];
#pragma unroll
      for (int s = 0; s < 2; ++s) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const float* at = &k[(16 * s + 8 * h + 2 * t) * ldr + nt * 8 + g];
          split_bf16(at[0], at[ldr], kh[s][h], kl[s][h]);
        }
      }
      float acc[2][4] = {};
#pragma unroll
      for (int b = 0; b < 3; ++b) {
        const int s = b == 2 ? 1 : 0, m = b > 0 ? 1 : 0;
        mma16816(acc[m], th[b], kh[s][0], kh[s][1]);
        mma16816(acc[m], th[b], kl[s][0], kl[s][1]);
        mma16816(acc[m], tl[b], kh[s][0], kh[s][1]);
      }
#pragma unroll
      for (int m = 0; m < 2; ++m) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          uint32_t hi, lo;
          split_bf16(acc[m][2 * h], acc[m][2 * h + 1], hi, lo);
          unsigned char* at = out + (size_t)(16 * m + 8 * h + g) * qk_row(dkp) + (nt * 8 + 2 * t) * 2;
          *reinterpret_cast<uint32_t*>(at + off_w(dkp, 0)) = hi;
          *reinterpret_cast<uint32_t*>(at + off_w(dkp, 1)) = lo;
        }
      }
    }
  }
  // U^T = V^T (T diag(beta))^T: 16 columns of V at a time, each read by one warp only
  {
    uint32_t bh[6][2], bl[6][2];  // (tokens 0-7, 8-15 from the first 16), (16-23, 24-31 from the first and the second 16)
#pragma unroll
    for (int b = 0; b < 6; ++b) {
      const int i = (b < 2 ? b : 2 + ((b - 2) >> 1)) * 8 + g, j0 = b >= 2 && (b & 1) ? 16 : 0;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int j = j0 + 8 * h + 2 * t;
        split_bf16(Ti[i * kLdT + j] * s_beta[j], Ti[i * kLdT + j + 1] * s_beta[j + 1], bh[b][h], bl[b][h]);
      }
    }
    unsigned char* values = a.g.values + ((size_t)chunk * a.g.heads + head) * a.g.v_bytes;
    for (int mt = warp; mt < a.g.n_slices * (kScanCols / 16); mt += 8) {
      const int c0 = mt * 16 + g;
      uint32_t vh[2][4], vl[2][4];
#pragma unroll
      for (int s = 0; s < 2; ++s) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {  // (column g, tokens 2t, 2t + 1), (g + 8, ..), (g, tokens 8 on), (g + 8, ..)
          const int col = c0 + (e & 1) * 8, tok = 16 * s + (e >> 1) * 8 + 2 * t;
          const float x = col < dv && tok < n ? a.v(it.x + tok, head)[col] : 0.f, y = col < dv && tok + 1 < n ? a.v(it.x + tok + 1, head)[col] : 0.f;
          split_bf16(x, y, vh[s][e], vl[s][e]);
        }
      }
      float* dst = reinterpret_cast<float*>(values + (size_t)(mt / (kScanCols / 16)) * kUSlice) + ((mt % (kScanCols / 16)) * 16 + g) * kUStride + 2 * t;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int s = 0; s < (nt < 2 ? 1 : 2); ++s) {
          const int b = nt < 2 ? nt : 2 + (nt - 2) * 2 + s;
          mma16816(acc, vh[s], bh[b][0], bh[b][1]);
          mma16816(acc, vh[s], bl[b][0], bl[b][1]);
          mma16816(acc, vl[s], bh[b][0], bh[b][1]);
        }
        *reinterpret_cast<float2*>(dst + nt * 8) = make_float2(acc[0], acc[1]);
        *reinterpret_cast<float2*>(dst + 8 * kUStride + nt * 8) = make_float2(acc[2], acc[3]);
      }
    }
  }
}

b200_status check(const b200_kv* kv, const GlaScratch& g, const DeltaCall& c, int total_rows) {
  if (c.layer < 0 || c.layer >= kv->cfg.n_layers || c.heads <= 0 || c.kv_heads <= 0 || c.heads % c.kv_heads != 0 || c.conv.taps < 1 ||
      kv->lay[c.layer].rec_elems < b200_delta_elems(c.heads, c.kv_heads, c.dk, c.dv, c.conv.taps)) {
    b200_set_error("delta rule: layer %d of the pool has no state of %d x %d x %d", c.layer, c.heads, c.dk, c.dv);
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (total_rows > g.max_rows || b200_delta_channels(c.heads, c.kv_heads, c.dk, c.dv) > (int)g.row_elems || c.heads > g.gate_heads) {
    b200_set_error("delta rule: %d rows of %d heads exceed the scratch", total_rows, c.heads);
    return B200_ERR_CAPACITY;
  }
  return B200_OK;
}

bool by_four(const b200_kv* kv, const DeltaCall& c) {
  return c.dk % 4 == 0 && c.dv % 4 == 0 && kv->lay[c.layer].rec_elems % 4 == 0 && (c.src.ws || c.src.y_stride % 4 == 0);
}
int row_stride(const DeltaCall& c) { return (b200_delta_channels(c.heads, c.kv_heads, c.dk, c.dv) + 3) / 4 * 4; }

}  // namespace

b200_status b200_delta_prep(b200_kv* kv, const GlaScratch& g, const DeltaCall& c, const int32_t* d_cu, const int32_t* d_row_to_req,
                            const int32_t* d_row_seq, const int32_t* d_pos, int total_rows, void* stream) {
  if (total_rows <= 0) return B200_OK;
  b200_status st = check(kv, g, c, total_rows);
  if (st != B200_OK) return st;
  PrepArgs a;
  a.c = c;
  a.c.conv.channels = b200_delta_channels(c.heads, c.kv_heads, c.dk, c.dv);
  a.c.conv.state = kv->dev.rec_pool + kv->lay[c.layer].rec_off + b200_delta_conv_off(c.heads, c.dk, c.dv);
  a.c.conv.slot_elems = kv->lay[c.layer].rec_elems;
  a.pool_state = kv->dev.state; a.cu = d_cu; a.row_to_req = d_row_to_req; a.row_seq = d_row_seq; a.pos = d_pos; a.max_seqs = kv->dev.max_seqs;
  a.rows = g.rows; a.stride = row_stride(c); a.gates = g.gates;
  a.q_scale = (float)(1.0 / std::sqrt((double)c.dk));
  const bool f32 = kv->dev.elem_bytes == 4, v4 = by_four(kv, c), many = total_rows >= 1024 && v4 && !f32 && c.conv.taps == 4;
  a.v_units = (c.heads * c.dv + (v4 ? 128 : 32) - 1) / (v4 ? 128 : 32);
  auto* kernel = f32 ? (v4 ? delta_prep_kernel<float, 4, 0, 1> : delta_prep_kernel<float, 1, 0, 1>)
                     : (v4 ? delta_prep_kernel<__nv_bfloat16, 4, 0, 1> : delta_prep_kernel<__nv_bfloat16, 1, 0, 1>);
  if (many) kernel = delta_prep_kernel<__nv_bfloat16, 4, 4, 4>;
  kernel<<<dim3(many ? (total_rows + 3) / 4 : total_rows, (2 * c.kv_heads + a.v_units + 1 + 7) / 8), 256, 0, (cudaStream_t)stream>>>(a, total_rows);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

b200_status b200_delta_run(b200_kv* kv, const GlaScratch& g, const DeltaCall& c, const int32_t* d_cu, const int32_t* d_row_seq, const int32_t* d_pos,
                           int n_req, int total_rows, bool chunked, void* stream) {
  if (n_req <= 0 || total_rows <= 0) return B200_OK;
  b200_status st = check(kv, g, c, total_rows);
  if (st != B200_OK) return st;
  const bool f32 = kv->dev.elem_bytes == 4;
  cudaStream_t s = (cudaStream_t)stream;
  Delta a{};
  Gla& z = a.g;
  z.d = kv->dev;
  z.state = kv->dev.rec_pool + kv->lay[c.layer].rec_off;
  z.rec_elems = kv->lay[c.layer].rec_elems;
  z.heads = c.heads; z.dk = c.dk; z.dv = c.dv; z.dkp = pad_channels(c.dk); z.dva = z.dvs = c.dv;
  z.src = c.src; z.norm = c.norm; z.eps = c.eps; z.out = c.out; z.out_stride = c.out_stride; z.cu = d_cu; z.row_seq = d_row_seq; z.pos = d_pos;
  z.n_req = n_req; z.total_rows = total_rows; z.chunks = g.chunks; z.values = g.values; z.o = g.o; z.plan = g.plan; z.first_chunk = g.first_chunk;
  z.chunk_bytes = delta_chunk_size(z.dkp);
  z.n_slices = slices_of(c.dv);
  z.v_bytes = z.n_slices * kUSlice;
  z.col_g = b200_delta_channels(c.heads, c.kv_heads, c.dk, c.dv);
  z.chunked = chunked && b200_gla_takes_chunks(c.dk, c.dv, kv->dev.elem_bytes);
  a.kv_heads = c.kv_heads; a.stride = row_stride(c); a.rows = g.rows; a.gates = g.gates;
  {
    const bool v4 = c.dv % 4 == 0 && z.rec_elems % 4 == 0 && (c.kv_heads * c.dk) % 2 == 0;
    const int vec = v4 ? 4 : 1;
    z.cols = std::min((c.dv + vec - 1) / vec, 256);
    z.groups = std::max(1, std::min(256 / z.cols, (c.dk + 7) / 8));
    const int need = z.cols * vec >= c.dv ? (c.dk + z.groups - 1) / z.groups : 1 << 20;  // state rows of a thread
    const size_t smem = sizeof(float) * (2 * (size_t)c.dk + 2 * (size_t)z.groups * z.cols * vec + c.dv + 4);
    if (smem > 200 * 1024) { b200_set_error("delta rule: head widths %d / %d are too large", c.dk, c.dv); return B200_ERR_UNSUPPORTED; }
    auto run = [&](auto* kernel) -> b200_status {
      if (smem > 48 * 1024) B200_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
      kernel<<<dim3(n_req, c.heads), (z.cols * z.groups + 31) / 32 * 32, smem, s>>>(a);
      B200_LAUNCH_CHECK();
      return B200_OK;
    };
    auto pick = [&](auto tag) -> b200_status {
      using T = decltype(tag);
      if (!v4) return need <= 16 ? run(delta_step_kernel<T, 1, 16>) : run(delta_step_kernel<T, 1, 0>);
      if (need <= 8) return run(delta_step_kernel<T, 4, 8>);
      if (need <= 16) return run(delta_step_kernel<T, 4, 16>);
      return need <= 32 ? run(delta_step_kernel<T, 4, 32>) : run(delta_step_kernel<T, 4, 0>);
    };
    st = f32 ? pick(float{}) : pick(__nv_bfloat16{});
    if (st != B200_OK) return st;
  }
  if (!z.chunked || total_rows <= n_req) return B200_OK;
  const int chunks = std::min(total_rows / kC + n_req, g.max_chunks);
  const size_t smem = sizeof(float) * (2 * (size_t)kC * (z.dkp + 8) + 2 * (size_t)kC * kLdT);
  static bool configured = false;
  if (!configured) {
    B200_CUDA_TRY(cudaFuncSetAttribute(delta_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024));
    configured = true;
  }
  delta_chunk_kernel<<<dim3(chunks, c.heads), 256, smem, s>>>(a);
  B200_LAUNCH_CHECK();
  if ((st = b200_gla_scan(z, n_req, true, s)) != B200_OK) return st;
  return b200_gla_out(z, chunks, by_four(kv, c) && c.out_stride % 4 == 0, s);
}
