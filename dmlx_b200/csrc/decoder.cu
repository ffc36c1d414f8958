// Configurable decoder stack over a packed ragged batch (model_step.cu packs it and reserves its pages).  Each layer says
// which mechanisms it has (b200_decoder_layer); the stack may run a range of layers several times with the same weights, each
// pass opening with x = W_in [x ; x0].
//
// An attention layer is six launches: q/k/v matmul; decoder_qkv_kernel (split-K finish, biases, per-head norms, q to the
// attention's operand, k and v straight into their pages); attention (attn_window.cu); o matmul; decoder_rows_kernel (split-K
// finish, post-norm, f32 residual add, and the norm or the [x ; x0] rows the next matmul reads); then the feed-forward's
// two matmuls around the SwiGLU epilogue and decoder_rows_kernel again.
//
// Latent attention: projection; latent_prep_kernel (attn_latent.cu); W_uk per head onto the queries; attention over the latents;
// W_uv per head.  Gated linear attention: projection; the kernels of gla.cu.  Where mixer and feed-forward run in parallel, the
// mixer's W_o and the dense feed-forward's W_down are one matmul over the concatenation [mixer output | SwiGLU output], and a
// single decoder_rows_kernel adds it, gathers the experts' rows, averages over depth and norms for the next layer.  Experts by
// token id are planned for all layers at the start of the step (moe.cu).
//
// A matrix memory beside attention shares its projection and W_o: gate matmul (f32 sums) and memory_gates_kernel, projection of both
// branches, decoder_qkv_conv(4)_kernel (convolution, norms, rotation, pages), attention, the kernels of gla.cu.  The branches' factors ride on
// the values and on the memory's output, so the product needs none.  Gated linear recurrence: projection, lru_prep_kernel, the blocks' gate
// matmuls with f32 sums, lru_scan_kernel (lru.cu).  Latent queries may take a detour over a latent of their own (one more norm and matmul), and
// a latent layer may read the pages of an earlier one.  A router's logits stay f32 sums, which route_src_kernel reads in place (moe.cu).
//
// With norms behind the sum decoder_rows_kernel scales the residual, adds, norms, and writes the result twice: as the residual and as the
// operand of the next matmul.
//
// Gated delta rule: projection; delta_prep_kernel; the kernels of delta.cu and gla.cu.  Where a sublayer reads h + conv(h), decoder_rows_kernel
// writes both in steps of single tokens; otherwise input_conv_kernel stands behind it.  A gate on a sublayer's result is a matmul from h whose
// partial sums wait aside (b200_qmm_deferred_aside) until decoder_rows_kernel multiplies its sigmoid in, ahead of the post-norm.
//
// The residual, every norm, the biases and the logits are f32; matrix operands are bf16, or f32 with B200_DT_F32 (the same
// kernels instantiated for float, matmuls through b200_qmm_f32, attention on CUDA cores).
//
// Matrices are padded with zero rows and columns to multiples of 64, so any width runs; the columns an activation row has
// behind its own width meet zero weights.
#include <cuda_bf16.h>

#include <algorithm>
#include <cmath>
#include <cstring>
#include <map>
#include <type_traits>
#include <vector>

#include "attn_latent.cuh"
#include "common.h"
#include "delta.cuh"
#include "gla.cuh"
#include "kv_pool.cuh"
#include "lru.cuh"
#include "model_step.cuh"
#include "moe.cuh"
#include "qmm.cuh"
#include "rows.cuh"
#include "short_conv.cuh"

namespace {

constexpr int kPageTokens = 32;     // of every pool
constexpr float kMemoryEps = 1e-6f;  // added to a matrix memory's denominator
constexpr double kLog2e = 1.4426950408889634;

int pad64(int n) { return (n + 63) / 64 * 64; }

// ---- between the matmuls ------------------------------------------------------------------------------------
struct RowArgs {
  int hidden;
  float eps;
  const uint32_t* tokens = nullptr;  // set: the row is the embedding of its token (x and x0 are written)
  const __nv_bfloat16* embed = nullptr;
  int vocab = 0;
  float embed_scale = 1.f;
  const __nv_bfloat16* pos_embed = nullptr;  // [max_positions][hidden], added to the embedding
  int max_positions = 0;
  MatSrc src;
  const float* src_scale = nullptr;  // factor per row on src (not on the experts)
  MatSrc gate;                    // with a bias: src and experts are multiplied by sigmoid(gate + gate_bias), ahead of the post-norm
  const float* gate_bias = nullptr;
  const float* post_w = nullptr;  // post-norm of the sublayer's output
  int replace = 0;                // x = src instead of x += src
  float* x = nullptr;
  float* x0 = nullptr;            // embedding output (null without a loop)
  const float* norm_w = nullptr;  // h = norm(x) * norm_w for the next matmul
  void* h = nullptr;
  int h_stride = 0;
  void* cat = nullptr;            // [x ; x0] for the loop's input matmul
  int cat_stride = 0;
  // experts: src also gets moe_w times the sum of the row's moe_k rows of moe_y
  const void* moe_y = nullptr;
  const int* moe_rows = nullptr;  // [row * moe_k + j] -> row of moe_y
  int moe_k = 0, moe_stride = 0;
  float moe_w = 0.f;
  const float* moe_wts = nullptr;  // [row * moe_k + j]: a weight of its own for each, instead of moe_w
  // norms behind the sum: x = norm(x_scale * x + src) * norm_w is the residual and what the next matmul reads
  float x_scale = 1.f;
  int norm_x = 0;
  int plain_h = 0;                // h = x without a norm
  // depth average: the result is kept as hist[n_hist], and x becomes sum_j depth[j] hist[j]
  const float* depth = nullptr;   // null for the embedding, which is kept as it is
  float* hist = nullptr;
  size_t hist_stride = 0;
  int n_hist = 0;
  // rows of single tokens: hc = h + conv(h), and the convolution's state moves on
  ShortConv conv;
  void* hc = nullptr;
  const int *pos = nullptr, *row_seq = nullptr, *pool_state = nullptr;
  int max_seqs = 0;
};

// x as a later kernel finds it in an operand of this type.
template <typename T>
__device__ __forceinline__ float as_stored(float x) {
  if constexpr (std::is_same_v<T, float>) return x;
  else return __bfloat162float(__float2bfloat16(x));
}

// One CTA per row: sublayer output -> residual stream -> what the next matmul reads.  NQ > 0: a thread keeps its NQ
// groups of VEC columns in registers and asks for the residual before the first reduction; NQ = 0: any width, the row
// waits in shared memory.  FEW: steps of few rows, bound by the latency of their loads, so more of them are in flight; only they may do the
// convolution of the coming sublayer.
constexpr int kStateAhead = 3;  // entries of its state that are asked for before the row's sums are known
template <typename T, int VEC, int NQ, bool FEW>
__global__ void __launch_bounds__(512, FEW ? 1 : 2) decoder_rows_kernel(RowArgs a) {
  extern __shared__ float row_sh[];
  __shared__ float part[32];
  __shared__ float4 part4[32];
  const int row = blockIdx.x, n = a.hidden / VEC;
  float* xr = a.x + (size_t)row * a.hidden;
  float* x0r = a.x0 ? a.x0 + (size_t)row * a.hidden : nullptr;
  Vec<VEC> keep[NQ > 0 ? NQ : 1];
  // visits the thread's groups; get/put move a group between them and registers or shared memory
  auto each = [&](auto f) {
    if constexpr (NQ > 0) {
#pragma unroll
      for (int k = 0; k < NQ; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
        if (i < n) f(i, k);
      }
    } else {
      for (int i = threadIdx.x; i < n; i += blockDim.x) f(i, 0);
    }
  };
  auto get = [&](int i, int k) -> Vec<VEC> {
    if constexpr (NQ > 0) return keep[k];
    else return load_vec<VEC>(row_sh + i * VEC);
  };
  auto put = [&](int i, int k, const Vec<VEC>& v) {
    if constexpr (NQ > 0) keep[k] = v;
    else store_vec<VEC>(row_sh + i * VEC, v);
  };
  auto value = [&](const MatSrc& src, int c) {
    if constexpr (FEW) return mat_value_ahead<T, VEC, 8>(src, row, c);
    else return mat_value<T, VEC>(src, row, c);
  };
  const int slot = FEW && a.hc ? a.row_seq[row] : 0;
  const bool conv = FEW && a.hc && slot >= 0 && slot < a.max_seqs && a.pool_state[ST_ERR] == 0;
  const int back = conv ? min(a.conv.taps - 1, a.pos[row]) : 0;
  float* state = conv ? a.conv.state + (size_t)slot * a.conv.slot_elems : nullptr;
  constexpr int kAhead = FEW && NQ > 0 ? kStateAhead : 0;
  Vec<VEC> old[kAhead > 0 ? NQ * kAhead : 1];
  if (kAhead > 0 && conv) {
    each([&](int i, int k) {
#pragma unroll
      for (int d = 0; d < kAhead; ++d)
        if (d + 1 < a.conv.taps) old[k * kAhead + d] = load_vec<VEC>(state + (size_t)d * a.conv.channels + i * VEC);
    });
  }
  float ss = 0.f, r_h = 0.f;
  // With a post-norm both norms come out of one round of sums: |x + r p|^2 = |x|^2 + 2 r x.p + r^2 |p|^2 for p = w y.
  const bool one_round = NQ > 0 && sizeof(T) == 2 && !a.tokens && a.post_w && a.norm_w && !a.replace && !a.depth && !a.norm_x && !a.plain_h && !a.cat;
  float4 sums = make_float4(0.f, 0.f, 0.f, 0.f);
  if (a.tokens) {
    const uint32_t tok = min(a.tokens[row], (uint32_t)(a.vocab - 1));
    const __nv_bfloat16* e = a.embed + (size_t)tok * a.hidden;
    each([&](int i, int k) {
      Vec<VEC> v = load_vec<VEC>(e + i * VEC);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v.v[j] *= a.embed_scale;
      if (a.pos_embed) {
        const Vec<VEC> p = load_vec<VEC>(a.pos_embed + (size_t)min(a.pos[row], a.max_positions - 1) * a.hidden + i * VEC);
#pragma unroll
        for (int j = 0; j < VEC; ++j) v.v[j] += p.v[j];
      }
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss += v.v[j] * v.v[j];
      put(i, k, v);
      store_vec<VEC>(xr + i * VEC, v);
      if (x0r) store_vec<VEC>(x0r + i * VEC, v);
      if (a.hist) store_vec<VEC>(a.hist + (size_t)row * a.hidden + i * VEC, v);
    });
  } else {
    float ys = 0.f;
    const float src_scale = a.src_scale ? a.src_scale[row] : 1.f;
    Vec<VEC> res[NQ > 0 ? NQ : 1];
    if (NQ > 0 && !a.replace) each([&](int i, int k) { res[k] = load_vec<VEC>(xr + i * VEC); });
    // rows that the matmuls wrote themselves are asked for at once
    constexpr bool kRowsAhead = NQ > 0 && !FEW;
    Raw<T, VEC> y_raw[kRowsAhead ? NQ : 1], z_raw[kRowsAhead ? NQ : 1];
    const T* y_row = kRowsAhead && !a.src.ws && a.src.y ? (const T*)a.src.y + (size_t)row * a.src.y_stride : nullptr;
    const T* z_row = kRowsAhead && !a.gate.ws && a.gate_bias ? (const T*)a.gate.y + (size_t)row * a.gate.y_stride : nullptr;
    if (y_row) each([&](int i, int k) { y_raw[k] = load_raw<T, VEC>(y_row + i * VEC); });
    if (z_row) each([&](int i, int k) { z_raw[k] = load_raw<T, VEC>(z_row + i * VEC); });
    each([&](int i, int k) {
      Vec<VEC> v;
      if (a.src.ws || a.src.y) {
        v = y_row ? widen<T, VEC>(y_raw[kRowsAhead ? k : 0]) : value(a.src, i * VEC);
#pragma unroll
        for (int j = 0; j < VEC; ++j) v.v[j] *= src_scale;
      } else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) v.v[j] = 0.f;
      }
      for (int m = 0; m < a.moe_k; ++m) {
        const Vec<VEC> e = load_vec<VEC>((const T*)a.moe_y + (size_t)a.moe_rows[row * a.moe_k + m] * a.moe_stride + i * VEC);
        const float w = a.moe_wts ? a.moe_wts[row * a.moe_k + m] : a.moe_w;
#pragma unroll
        for (int j = 0; j < VEC; ++j) v.v[j] = fmaf(w, e.v[j], v.v[j]);
      }
      if (a.gate_bias) {
        const Vec<VEC> z = z_row ? widen<T, VEC>(z_raw[kRowsAhead ? k : 0]) : value(a.gate, i * VEC), b = load_vec<VEC>(a.gate_bias + i * VEC);
#pragma unroll
        for (int j = 0; j < VEC; ++j) v.v[j] *= sigmoid_for<T>(z.v[j] + b.v[j]);
      }
      if (one_round) {
        const Vec<VEC> w = load_vec<VEC>(a.post_w + i * VEC), x = res[NQ > 0 ? k : 0];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          sums.x = fmaf(v.v[j], v.v[j], sums.x);
          v.v[j] *= w.v[j];
          sums.y = fmaf(x.v[j], x.v[j], sums.y);
          sums.z = fmaf(x.v[j], v.v[j], sums.z);
          sums.w = fmaf(v.v[j], v.v[j], sums.w);
        }
      } else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) ys += v.v[j] * v.v[j];
      }
      put(i, k, v);
    });
    if (one_round) {
      sums = block_sum4(sums, part4);
      const float r = 1.0f / sqrtf(sums.x / (float)a.hidden + a.eps);
      r_h = 1.0f / sqrtf(fmaxf(fmaf(r, fmaf(r, sums.w, 2.f * sums.z), sums.y), 0.f) / (float)a.hidden + a.eps);
      each([&](int i, int k) {
        Vec<VEC> v = get(i, k), x = res[NQ > 0 ? k : 0];
#pragma unroll
        for (int j = 0; j < VEC; ++j) v.v[j] = fmaf(r, v.v[j], x.v[j]);
        put(i, k, v);
        store_vec<VEC>(xr + i * VEC, v);
      });
    } else {
      const float r = a.post_w ? 1.0f / sqrtf(block_sum(ys, part) / (float)a.hidden + a.eps) : 1.f;
      each([&](int i, int k) {
        Vec<VEC> v = get(i, k);
        if (a.post_w) {
          const Vec<VEC> w = load_vec<VEC>(a.post_w + i * VEC);
#pragma unroll
          for (int j = 0; j < VEC; ++j) v.v[j] *= r * w.v[j];
        }
        if (!a.replace) {
          Vec<VEC> x;
          if constexpr (NQ > 0) x = res[k];
          else x = load_vec<VEC>(xr + i * VEC);
#pragma unroll
          for (int j = 0; j < VEC; ++j) v.v[j] = fmaf(a.x_scale, x.v[j], v.v[j]);
        }
        if (a.depth) {
          float* hr = a.hist + (size_t)row * a.hidden + i * VEC;
          store_vec<VEC>(hr + a.n_hist * a.hist_stride, v);
          const float own = a.depth[a.n_hist];
#pragma unroll
          for (int j = 0; j < VEC; ++j) v.v[j] *= own;
#pragma unroll 4
          for (int d = 0; d < a.n_hist; ++d) {
            const Vec<VEC> x = load_vec<VEC>(hr + d * a.hist_stride);
            const float w = a.depth[d];
#pragma unroll
            for (int j = 0; j < VEC; ++j) v.v[j] = fmaf(w, x.v[j], v.v[j]);
          }
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += v.v[j] * v.v[j];
        put(i, k, v);
        if (!a.norm_x) store_vec<VEC>(xr + i * VEC, v);
      });
    }
  }
  if (a.plain_h) {
    T* hr = (T*)a.h + (size_t)row * a.h_stride;
    each([&](int i, int k) { store_vec<VEC>(hr + i * VEC, get(i, k)); });
  }
  if (a.norm_w) {
    const float r = one_round ? r_h : 1.0f / sqrtf(block_sum(ss, part) / (float)a.hidden + a.eps);
    T* hr = (T*)a.h + (size_t)row * a.h_stride;
    each([&](int i, int k) {
      Vec<VEC> v = get(i, k);
      const Vec<VEC> w = load_vec<VEC>(a.norm_w + i * VEC);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v.v[j] *= r * w.v[j];
      store_vec<VEC>(hr + i * VEC, v);
      if (conv) {
        float* entry = state + i * VEC;
        Vec<VEC> own, acc{};
#pragma unroll
        for (int j = 0; j < VEC; ++j) own.v[j] = as_stored<T>(v.v[j]);
        Vec<VEC> carried = own;  // entries move up by one
        auto step = [&](int d, const Vec<VEC>& u) {
          store_vec<VEC>(entry + (size_t)(d - 1) * a.conv.channels, carried);
          carried = u;
          if (d <= back) {
            const Vec<VEC> tap = load_vec<VEC>(a.conv.w + (size_t)(a.conv.taps - 1 - d) * a.conv.channels + i * VEC);
#pragma unroll
            for (int j = 0; j < VEC; ++j) acc.v[j] = fmaf(tap.v[j], u.v[j], acc.v[j]);
          }
        };
#pragma unroll
        for (int d = 1; d <= kAhead; ++d)
          if (d < a.conv.taps) step(d, old[k * kAhead + d - 1]);
        for (int d = kAhead + 1; d < a.conv.taps; ++d) step(d, load_vec<VEC>(entry + (size_t)(d - 1) * a.conv.channels));
        const Vec<VEC> tap = load_vec<VEC>(a.conv.w + (size_t)(a.conv.taps - 1) * a.conv.channels + i * VEC);
#pragma unroll
        for (int j = 0; j < VEC; ++j) acc.v[j] = own.v[j] + fmaf(tap.v[j], own.v[j], acc.v[j]);
        store_vec<VEC>((T*)a.hc + (size_t)row * a.h_stride + i * VEC, acc);
      }
      if (a.norm_x) store_vec<VEC>(xr + i * VEC, v);
    });
  }
  if (a.cat) {
    T* cr = (T*)a.cat + (size_t)row * a.cat_stride;
    each([&](int i, int k) {
      store_vec<VEC>(cr + i * VEC, get(i, k));
      store_vec<VEC>(cr + a.hidden + i * VEC, load_vec<VEC>(x0r + i * VEC));  // (an embedding row was written by this thread)
    });
  }
}

template <typename T, bool FEW>
void (*rows_kernel(int vec, int nq))(RowArgs) {
  if (vec == 1) return decoder_rows_kernel<T, 1, 0, FEW>;
  return nq <= 1 ? decoder_rows_kernel<T, 4, 1, FEW> : (nq <= 2 ? decoder_rows_kernel<T, 4, 2, FEW> : (nq <= 4 ? decoder_rows_kernel<T, 4, 4, FEW> : decoder_rows_kernel<T, 4, 0, FEW>));
}

// hc = h + conv(h) over the rows of a step, portions of any length.  One thread per (R rows, VEC channels).
struct InputConvArgs {
  ShortConv conv;
  const void* h;
  void* hc;
  int hidden, stride, max_seqs;
  const int *pool_state, *cu, *row_to_req, *row_seq, *pos;
};

template <typename T, int VEC, int TAPS, int R>
__global__ void __launch_bounds__(256) input_conv_kernel(InputConvArgs a, int rows) {
  const int begin = blockIdx.x * R, end = min(begin + R, rows), ch = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (ch >= a.hidden || a.pool_state[ST_ERR] != 0) return;
  auto value = [&](int row, int col) { return load_vec<VEC>((const T*)a.h + (size_t)row * a.stride + col); };
  auto put = [&](int row, Vec<VEC> y) {
    const Vec<VEC> x = value(row, ch);
#pragma unroll
    for (int e = 0; e < VEC; ++e) y.v[e] += x.v[e];
    store_vec<VEC>((T*)a.hc + (size_t)row * a.stride + ch, y);
  };
  if constexpr (R > 1 && TAPS > 0) {
    if (begin + R <= rows && a.row_to_req[begin] == a.row_to_req[begin + R - 1] && begin - a.cu[a.row_to_req[begin]] >= TAPS - 1) {
      Vec<VEC> y[R];
      conv_values_inside<TAPS, R, VEC>(a.conv, value, begin, ch, y);
#pragma unroll
      for (int r = 0; r < R; ++r) put(begin + r, y[r]);
      return;
    }
  }
  for (int first = begin; first < end; ++first) {
    const int req = a.row_to_req[first], r0 = a.cu[req], count = a.cu[req + 1] - r0, slot = a.row_seq[first];
    if (slot < 0 || slot >= a.max_seqs) continue;
    const int n = conv_rows(a.conv, first - r0, count);
    for (int row = first; row < first + n; ++row) put(row, conv_value<VEC>(a.conv, value, row, row - r0, a.pos[row], slot, ch));
    if (first == r0) conv_update<VEC>(a.conv, value, r0, count, slot, ch);
  }
}

b200_status launch_input_conv(const InputConvArgs& a, int rows, bool f32, cudaStream_t s) {
  const bool v4 = a.hidden % 4 == 0 && a.stride % 4 == 0 && a.conv.slot_elems % 4 == 0, many = rows >= 256 && v4 && !f32;
  const int groups = v4 ? a.hidden / 4 : a.hidden, threads = std::min(256, (groups + 31) / 32 * 32);
  auto run = [&](auto* kernel, int per) -> b200_status {
    kernel<<<dim3((rows + per - 1) / per, (groups + threads - 1) / threads), threads, 0, s>>>(a, rows);
    B200_LAUNCH_CHECK();
    return B200_OK;
  };
  using B = __nv_bfloat16;
  if (many && a.conv.taps == 2) return run(input_conv_kernel<B, 4, 2, 4>, 4);
  if (many && a.conv.taps == 3) return run(input_conv_kernel<B, 4, 3, 4>, 4);
  if (many && a.conv.taps == 4) return run(input_conv_kernel<B, 4, 4, 4>, 4);
  if (f32) return v4 ? run(input_conv_kernel<float, 4, 0, 1>, 1) : run(input_conv_kernel<float, 1, 0, 1>, 1);
  return v4 ? run(input_conv_kernel<B, 4, 0, 1>, 1) : run(input_conv_kernel<B, 1, 0, 1>, 1);
}

// Rows idx[r] of x, normalised, as the head's operand.
template <typename T>
__global__ void __launch_bounds__(256) decoder_final_kernel(const float* __restrict__ x, const int* __restrict__ idx, const float* __restrict__ w,
                                                            T* __restrict__ out, int hidden, int out_stride, float eps) {
  __shared__ float part[32];
  const float* xr = x + (size_t)max(idx[blockIdx.x], 0) * hidden;
  float ss = 0.f;
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) ss += xr[c] * xr[c];
  const float r = 1.0f / sqrtf(block_sum(ss, part) / (float)hidden + eps);
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) st(out + (size_t)blockIdx.x * out_stride + c, xr[c] * r * w[c]);
}

__global__ void __launch_bounds__(256) decoder_logits_kernel(MatSrc src, float* __restrict__ logits, int vocab) {
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c < vocab) logits[(size_t)blockIdx.y * vocab + c] = mat_value<float, 1>(src, blockIdx.y, c).v[0];
}

// ---- between the q/k/v projection and attention ---------------------------------------------------------------
struct QkvArgs {
  KvDev d;
  KvLayerDev L;
  MatSrc src;
  const float* bias;  // [q | k | v] columns, null without biases
  int hq, qk_norm;
  float eps;
  void* q;
  int q_stride;
  const int *pos, *row_seq;
  // convolution, weights of the q and k norms, rotation of the first `rot` dimensions, factor on v: decoder_qkv_conv_kernel
  const int *cu = nullptr, *row_to_req = nullptr;
  ShortConv conv;  // channels as in the projection's columns
  const float *q_norm = nullptr, *k_norm = nullptr;
  const float2* rotation = nullptr;
  int rot = 0, halves = 0;
  float v_scale = 1.f;
  // norms over the whole projection, query temperature, queries alone: decoder_qkv_row_kernel
  bool norm_row = false, keys = true;
  float temp_coef = 0.f;
  int temp_every = 0;  // 0: none
};

// Where key or value head `head` of a row lives in its page; null when the step's reservation failed (nothing is written then, the
// error word is set).
template <typename T>
__device__ __forceinline__ T* page_row(const QkvArgs& a, int row, int head, bool is_v) {
  const int pos = a.pos[row], seq = a.row_seq[row];
  const int page_idx = pos / kPageTokens, slot = pos % kPageTokens;
  if (seq < 0 || seq >= a.d.max_seqs || page_idx >= min(a.d.seq_pages[seq], a.d.max_pages_per_seq)) return nullptr;
  const int page = a.d.block_table[(size_t)seq * a.d.max_pages_per_seq + page_idx];
  char* pool = is_v ? (char*)a.d.v_pool + a.L.v_off : (char*)a.d.k_pool + a.L.k_off;
  return (T*)pool + (((size_t)page * a.L.heads + head) * kPageTokens + slot) * (size_t)(is_v ? a.L.vd : a.L.kd);
}

// One warp per (row, head); q heads, then k heads, then v heads.  Grid y covers the heads, eight at a time.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) decoder_qkv_kernel(QkvArgs a) {
  constexpr int KEEP = VEC == 4 ? 2 : 4;  // passes of 32 x VEC columns kept in registers; wider heads are read again
  const int row = blockIdx.x, lane = threadIdx.x & 31, H = a.L.heads;
  const int u = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (u >= a.hq + 2 * H) return;
  const bool is_q = u < a.hq, is_v = u >= a.hq + H;
  const int head = is_q ? u : (is_v ? u - a.hq - H : u - a.hq);
  const int dim = is_v ? a.L.value_dim : a.L.key_dim, width = is_v ? a.L.vd : a.L.kd;
  const int n0 = is_v ? (a.hq + H) * a.L.key_dim + head * dim : u * dim;
  T* dst = nullptr;
  if (is_q) {
    dst = (T*)a.q + (size_t)row * a.q_stride + (size_t)head * a.L.kd;
  } else {
    dst = page_row<T>(a, row, head, is_v);
    if (!dst) return;
  }
  auto value = [&](int c) {
    Vec<VEC> v = mat_value<T, VEC>(a.src, row, n0 + c);
    if (a.bias) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] += a.bias[n0 + c + e];
    }
    return v;
  };
  Vec<VEC> keep[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (i * 32 + lane) * VEC;
    if (c < dim) {
      keep[i] = value(c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += keep[i].v[e] * keep[i].v[e];
    }
  }
  for (int c = (KEEP * 32 + lane) * VEC; c < dim; c += 32 * VEC) {
    const Vec<VEC> v = value(c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += v.v[e] * v.v[e];
  }
  float r = 1.f;
  if (a.qk_norm && !is_v) r = 1.0f / sqrtf(warp_sum(ss) / (float)dim + a.eps);
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (i * 32 + lane) * VEC;
    if (c < dim) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) keep[i].v[e] *= r;
      store_vec<VEC>(dst + c, keep[i]);
    }
  }
  for (int c = (KEEP * 32 + lane) * VEC; c < dim; c += 32 * VEC) {
    Vec<VEC> v = value(c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] *= r;
    store_vec<VEC>(dst + c, v);
  }
  for (int c = dim + lane; c < width; c += 32) st(dst + c, 0.f);
}

// The same with everything a design may put between projection and attention: bias, convolution over the tokens before, norm with a
// weight, rotation.  One warp per (row, head), the head's row in shared memory; the warp of a request's first row also takes the rows
// that read the convolution's state (short_conv.cuh).
template <typename T, int VEC>
__global__ void __launch_bounds__(256) decoder_qkv_conv_kernel(QkvArgs a) {
  extern __shared__ float row_sh[];
  const int first = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, H = a.L.heads, u = blockIdx.y * 8 + warp;
  if (u >= a.hq + 2 * H || a.d.state[ST_ERR] != 0) return;
  const bool is_q = u < a.hq, is_v = u >= a.hq + H;
  const int head = is_q ? u : (is_v ? u - a.hq - H : u - a.hq);
  const int dim = is_v ? a.L.value_dim : a.L.key_dim, width = is_v ? a.L.vd : a.L.kd;
  const int n0 = is_v ? (a.hq + H) * a.L.key_dim + head * dim : u * dim;
  float* sh = row_sh + warp * max(a.L.key_dim, a.L.value_dim);
  const int req = a.row_to_req[first], r0 = a.cu[req], count = a.cu[req + 1] - r0, slot = a.row_seq[first];
  if (slot < 0 || slot >= a.d.max_seqs) return;
  auto value = [&](int row, int c) {
    Vec<VEC> v = mat_value<T, VEC>(a.src, row, c);
    if (a.bias) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] += a.bias[c + e];
    }
    return v;
  };
  const int n = conv_rows(a.conv, first - r0, count);
  const float* norm = is_q ? a.q_norm : (is_v ? nullptr : a.k_norm);
  for (int row = first; row < first + n; ++row) {
    T* dst = is_q ? (T*)a.q + (size_t)row * a.q_stride + (size_t)head * a.L.kd : page_row<T>(a, row, head, is_v);
    if (!dst) return;
    float ss = 0.f;
    for (int c = lane * VEC; c < dim; c += 32 * VEC) {
      const Vec<VEC> v = a.conv.taps > 0 ? conv_value<VEC>(a.conv, value, row, row - r0, a.pos[row], slot, n0 + c) : value(row, n0 + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += v.v[e] * v.v[e];
      store_vec<VEC>(sh + c, v);
    }
    float r = is_v ? a.v_scale : 1.f;
    if (a.qk_norm && !is_v) r = 1.0f / sqrtf(warp_sum(ss) / (float)dim + a.eps);
    __syncwarp();
    auto at = [&](int c) { return norm ? sh[c] * r * norm[c] : sh[c] * r; };
    const int rot = is_v ? 0 : a.rot;
    for (int i = lane; i < rot / 2; i += 32) {
      const int c0 = a.halves ? i : 2 * i, c1 = a.halves ? i + rot / 2 : 2 * i + 1;
      const float2 cs = a.rotation[(size_t)row * (rot / 2) + i];
      const float x = at(c0), y = at(c1);
      st(dst + c0, x * cs.x - y * cs.y);
      st(dst + c1, y * cs.x + x * cs.y);
    }
    for (int c = rot + lane; c < width; c += 32) st(dst + c, c < dim ? at(c) : 0.f);
    __syncwarp();
  }
  if (first == r0 && a.conv.taps > 1)
    for (int c = lane * VEC; c < dim; c += 32 * VEC) conv_update<VEC>(a.conv, value, r0, count, slot, n0 + c);
}

// The same for four taps and heads up to KEEP * 128 wide, R rows per warp: a head's row stays in registers but for the columns that are
// rotated, and rows of one request that lie next to each other share the loads of their inputs and of the weights.
template <typename T, int KEEP, int R>
__global__ void __launch_bounds__(256, KEEP == 1 ? 3 : 2) decoder_qkv_conv4_kernel(QkvArgs a, int rows) {
  extern __shared__ float row_sh[];  // [warp][rot]
  const int begin = blockIdx.x * R, end = min(begin + R, rows);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, H = a.L.heads, u = blockIdx.y * 8 + warp;
  if (u >= a.hq + 2 * H || a.d.state[ST_ERR] != 0) return;
  const bool is_q = u < a.hq, is_v = u >= a.hq + H;
  const int head = is_q ? u : (is_v ? u - a.hq - H : u - a.hq);
  const int dim = is_v ? a.L.value_dim : a.L.key_dim, width = is_v ? a.L.vd : a.L.kd;
  const int n0 = is_v ? (a.hq + H) * a.L.key_dim + head * dim : u * dim;
  const int rot = is_v ? 0 : a.rot, half = rot / 2;
  float* sh = row_sh + warp * a.rot;
  const float* norm = is_q ? a.q_norm : (is_v ? nullptr : a.k_norm);
  auto value = [&](int row, int c) {
    Vec<4> v = mat_value<T, 4>(a.src, row, c);
    if (a.bias) {
#pragma unroll
      for (int e = 0; e < 4; ++e) v.v[e] += a.bias[c + e];
    }
    return v;
  };
  auto place = [&](int row) { return is_q ? (T*)a.q + (size_t)row * a.q_stride + (size_t)head * a.L.kd : page_row<T>(a, row, head, is_v); };
  const bool by_four = a.halves && half % 4 == 0;
  auto finish = [&](int row, Vec<4> (&x)[KEEP], T* dst) {  // norm, rotation, store
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      if ((k * 32 + lane) * 4 < dim) {
#pragma unroll
        for (int e = 0; e < 4; ++e) ss += x[k].v[e] * x[k].v[e];
      }
    }
    float r = is_v ? a.v_scale : 1.f;
    if (a.qk_norm && !is_v) r = 1.0f / sqrtf(warp_sum(ss) / (float)dim + a.eps);
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = (k * 32 + lane) * 4;
      if (c < dim) {
        Vec<4> f{{1.f, 1.f, 1.f, 1.f}};
        if (norm) f = load_vec<4>(norm + c);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          x[k].v[e] *= r * f.v[e];
          if (c + e < rot) sh[c + e] = x[k].v[e];
        }
      }
    }
    __syncwarp();
    if (dst) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int c = (k * 32 + lane) * 4;
        if (c < dim) {
          if (by_four) {
            if (c < rot) {
              const bool up = c >= half;
              const int i = up ? c - half : c;
              const Vec<4> other = load_vec<4>(sh + (up ? i : c + half));
              const float* cs = reinterpret_cast<const float*>(a.rotation + (size_t)row * half + i);
              const Vec<4> lo = load_vec<4>(cs), hi = load_vec<4>(cs + 4);  // cosine, sine, cosine, ..
              const float sign = up ? 1.f : -1.f;
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const Vec<4>& v = e < 2 ? lo : hi;
                x[k].v[e] = fmaf(sign * v.v[(2 * e + 1) & 3], other.v[e], x[k].v[e] * v.v[(2 * e) & 3]);
              }
            }
            store_vec<4>(dst + c, x[k]);
            continue;
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = c + e;
            if (i < rot) {
              const bool up = a.halves ? i >= half : (i & 1);
              const int other = a.halves ? (up ? i - half : i + half) : i ^ 1;
              const float2 cs = a.rotation[(size_t)row * half + (a.halves ? (up ? i - half : i) : i >> 1)];
              x[k].v[e] = fmaf(up ? cs.y : -cs.y, sh[other], x[k].v[e] * cs.x);
            }
          }
          store_vec<4>(dst + c, x[k]);
        }
      }
      for (int c = dim + lane; c < width; c += 32) st(dst + c, 0.f);
    }
    __syncwarp();
  };
  if constexpr (R > 1) {
    if (begin + R <= rows && a.row_to_req[begin] == a.row_to_req[begin + R - 1] && begin - a.cu[a.row_to_req[begin]] >= 3) {
      Vec<4> x[KEEP][R];
      T* dst[R];
#pragma unroll
      for (int r = 0; r < R; ++r) dst[r] = place(begin + r);
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int c = (k * 32 + lane) * 4;
        if (c < dim) {
          if (a.src.ws || a.bias) {
            conv_values_inside<4, R, 4>(a.conv, value, begin, n0 + c, x[k]);
          } else {  // rows the matmul wrote itself
            const T* y = (const T*)a.src.y + (size_t)begin * a.src.y_stride;
            conv_values_inside<4, R, 4>(a.conv, [&](int row, int col) { return load_vec<4>(y + (row - begin) * a.src.y_stride + col); }, begin, n0 + c, x[k]);
          }
        }
      }
#pragma unroll
      for (int r = 0; r < R; ++r) {
        Vec<4> row[KEEP];
#pragma unroll
        for (int k = 0; k < KEEP; ++k) row[k] = x[k][r];
        finish(begin + r, row, dst[r]);
      }
      return;
    }
  }
  for (int first = begin; first < end; ++first) {
    const int req = a.row_to_req[first], r0 = a.cu[req], count = a.cu[req + 1] - r0, slot = a.row_seq[first];
    if (slot < 0 || slot >= a.d.max_seqs) continue;
    const int n = conv_rows(a.conv, first - r0, count);
    for (int row = first; row < first + n; ++row) {
      const int pos = a.pos[row];
      Vec<4> x[KEEP];
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int c = (k * 32 + lane) * 4;
        if (c < dim) x[k] = conv_value<4>(a.conv, value, row, row - r0, pos, slot, n0 + c);
      }
      finish(row, x, place(row));
    }
    if (first == r0)
      for (int c = lane * 4; c < dim; c += 128) conv_update<4>(a.conv, value, r0, count, slot, n0 + c);
  }
}

// The same where a row's norms span all heads of q and of k: one CTA per row, which waits in shared memory for its sums of squares.  The queries are
// also scaled by a temperature that grows with the position; without keys there are queries only.
template <typename T, int VEC, int THREADS>
__global__ void __launch_bounds__(THREADS, 1024 / THREADS) decoder_qkv_row_kernel(QkvArgs a) {
  extern __shared__ __align__(16) float row_sh[];
  __shared__ float part[32];
  const int row = blockIdx.x, H = a.keys ? a.L.heads : 0, dim = a.L.key_dim, nq = a.hq * dim, nqk = nq + H * dim, all = nqk + H * a.L.value_dim;
  const int pos = a.pos[row];
  T *q = (T*)a.q + (size_t)row * a.q_stride, *kr = nullptr, *vr = nullptr;
  if (a.keys) {
    kr = page_row<T>(a, row, 0, false);
    if (!kr) return;
    vr = page_row<T>(a, row, 0, true);
  }
  const size_t k_head = (size_t)kPageTokens * a.L.kd, v_head = (size_t)kPageTokens * a.L.vd;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * VEC; c < all; c += THREADS * VEC) {
    Vec<VEC> v;
    if constexpr (THREADS > 256) v = mat_value_ahead<T, VEC, 8>(a.src, row, c);
    else v = mat_value<T, VEC>(a.src, row, c);
    if (a.bias) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] += a.bias[c + e];
    }
    if (c >= nqk) {
      const int head = (c - nqk) / a.L.value_dim;
      store_vec<VEC>(vr + head * v_head + (c - nqk - head * a.L.value_dim), v);
      continue;
    }
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) s += v.v[e] * v.v[e];
    if (c < nq) sq += s;
    else sk += s;
    store_vec<VEC>(row_sh + c, v);
  }
  float rq = 1.f, rk = 1.f;
  if (a.norm_row) {
    rq = 1.0f / sqrtf(block_sum(sq, part) / (float)nq + a.eps);
    __syncthreads();
    if (a.keys) rk = 1.0f / sqrtf(block_sum(sk, part) / (float)(nqk - nq) + a.eps);
  }
  if (a.temp_every > 0) rq *= 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every + 1));
  for (int c = threadIdx.x * VEC; c < nqk; c += THREADS * VEC) {  // (a thread reads what it wrote)
    const bool is_q = c < nq;
    const int k = is_q ? c : c - nq, head = k / dim;
    Vec<VEC> v = load_vec<VEC>(row_sh + c);
    const float* w = is_q ? a.q_norm : a.k_norm;
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] *= (is_q ? rq : rk) * (w ? w[k + e] : 1.f);
    store_vec<VEC>((is_q ? q + (size_t)head * a.L.kd : kr + head * k_head) + (k - head * dim), v);
  }
  for (int i = threadIdx.x; i < (a.hq + H) * (a.L.kd - dim); i += THREADS) {  // padding behind a head
    const int u = i / (a.L.kd - dim), c = dim + i - u * (a.L.kd - dim);
    st((u < a.hq ? q + (size_t)u * a.L.kd : kr + (u - a.hq) * k_head) + c, 0.f);
  }
  for (int i = threadIdx.x; i < H * (a.L.vd - a.L.value_dim); i += THREADS) {
    const int u = i / (a.L.vd - a.L.value_dim);
    st(vr + u * v_head + a.L.value_dim + i - u * (a.L.vd - a.L.value_dim), 0.f);
  }
}

b200_status launch_qkv(const QkvArgs& a, int rows, cudaStream_t s) {
  if (a.norm_row || a.temp_every > 0 || !a.keys) {
    const bool vec = a.L.key_dim % 4 == 0 && a.L.value_dim % 4 == 0 && (a.src.ws || a.src.y_stride % 4 == 0);
    const size_t smem = sizeof(float) * (a.hq + (a.keys ? a.L.heads : 0)) * (size_t)a.L.key_dim;
    if (smem > 200 * 1024) { b200_set_error("decoder: %d heads of %d are too wide for a row's norm", a.hq, a.L.key_dim); return B200_ERR_UNSUPPORTED; }
    const bool few = rows < 512;  // (one block per SM at most: more threads per row)
    auto* kernel = a.d.elem_bytes == 4 ? (vec ? decoder_qkv_row_kernel<float, 4, 256> : decoder_qkv_row_kernel<float, 1, 256>)
                                       : (vec ? decoder_qkv_row_kernel<__nv_bfloat16, 4, 256> : decoder_qkv_row_kernel<__nv_bfloat16, 1, 256>);
    if (few) kernel = a.d.elem_bytes == 4 ? (vec ? decoder_qkv_row_kernel<float, 4, 1024> : decoder_qkv_row_kernel<float, 1, 1024>)
                                          : (vec ? decoder_qkv_row_kernel<__nv_bfloat16, 4, 1024> : decoder_qkv_row_kernel<__nv_bfloat16, 1, 1024>);
    if (smem > 48 * 1024) B200_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kernel<<<rows, few ? 1024 : 256, smem, s>>>(a);
    B200_LAUNCH_CHECK();
    return B200_OK;
  }
  if (a.conv.taps > 0 || a.q_norm || a.rot > 0 || a.v_scale != 1.f) {
    const bool vec = a.L.key_dim % 4 == 0 && a.L.value_dim % 4 == 0 && (a.src.ws || a.src.y_stride % 4 == 0) && a.conv.slot_elems % 4 == 0 &&
                     a.conv.channels % 4 == 0;
    if (vec && a.conv.taps == 4 && !a.conv.bias && a.L.key_dim <= 256 && a.L.value_dim <= 256) {
      const bool narrow = a.L.key_dim <= 128 && a.L.value_dim <= 128, many = rows >= 1024;
      auto run = [&](auto* kernel, int per) {
        kernel<<<dim3((rows + per - 1) / per, (a.hq + 2 * a.L.heads + 7) / 8), 256, sizeof(float) * 8 * std::max(a.rot, 1), s>>>(a, rows);
      };
      auto pick = [&](auto tag) {
        using T = decltype(tag);
        if (many) narrow ? run(decoder_qkv_conv4_kernel<T, 1, 4>, 4) : run(decoder_qkv_conv4_kernel<T, 2, 4>, 4);
        else narrow ? run(decoder_qkv_conv4_kernel<T, 1, 1>, 1) : run(decoder_qkv_conv4_kernel<T, 2, 1>, 1);
      };
      if (a.d.elem_bytes == 4) pick(float{});
      else pick(__nv_bfloat16{});
      B200_LAUNCH_CHECK();
      return B200_OK;
    }
    const size_t smem = sizeof(float) * 8 * std::max(a.L.key_dim, a.L.value_dim);
    if (smem > 200 * 1024) { b200_set_error("decoder: head widths %d / %d are too large", a.L.key_dim, a.L.value_dim); return B200_ERR_UNSUPPORTED; }
    auto* kernel = a.d.elem_bytes == 4 ? (vec ? decoder_qkv_conv_kernel<float, 4> : decoder_qkv_conv_kernel<float, 1>)
                                       : (vec ? decoder_qkv_conv_kernel<__nv_bfloat16, 4> : decoder_qkv_conv_kernel<__nv_bfloat16, 1>);
    if (smem > 48 * 1024) B200_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kernel<<<dim3(rows, (a.hq + 2 * a.L.heads + 7) / 8), 256, smem, s>>>(a);
    B200_LAUNCH_CHECK();
    return B200_OK;
  }
  const bool v4 = a.L.key_dim % 4 == 0 && a.L.value_dim % 4 == 0 && a.src.y_stride % 4 == 0;
  auto* kernel = a.d.elem_bytes == 4 ? (v4 ? decoder_qkv_kernel<float, 4> : decoder_qkv_kernel<float, 1>)
                                     : (v4 ? decoder_qkv_kernel<__nv_bfloat16, 4> : decoder_qkv_kernel<__nv_bfloat16, 1>);
  kernel<<<dim3(rows, (a.hq + 2 * a.L.heads + 7) / 8), 256, 0, s>>>(a);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

struct HostTensor { std::vector<uint16_t> bits; };

float bf16_to_f(uint16_t b) {
  const uint32_t u = (uint32_t)b << 16;
  float f;
  std::memcpy(&f, &u, 4);
  return f;
}

const char* kTensorNames[] = {"q", "k", "v", "o", "gate", "up", "down", "head", "loop input", "embedding", "q bias", "k bias", "v bias",
                              "sink", "norm 1", "norm 2", "post-norm 1", "post-norm 2", "final norm", "latent", "latent norm", "key expansion",
                              "value expansion", "output gate", "decay 1", "decay 2", "decay bias", "head norm", "expert gate", "expert up",
                              "expert down", "depth weights", "query latent", "query latent norm", "q norm", "k norm", "q convolution",
                              "k convolution", "v convolution", "memory q", "memory k", "memory v", "memory output gate", "memory output",
                              "memory input gate", "memory forget gate", "memory input gate bias", "memory forget gate bias", "memory norm",
                              "lru branch", "lru branch bias", "lru input", "lru input bias", "lru convolution", "lru convolution bias",
                              "lru decay gate", "lru decay gate bias", "lru input gate", "lru input gate bias", "lru lambda", "router",
                              "positions", "distance table", "input convolution 1", "input convolution 2", "result gate 1", "result gate 2",
                              "result gate bias 1", "result gate bias 2", "beta", "decay", "decay rate", "decay bias", "shared expert gate"};
static_assert(sizeof(kTensorNames) / sizeof(kTensorNames[0]) == B200_DEC_LAST_TENSOR + 1, "a name per tensor");

}  // namespace

struct b200_decoder : b200_model {
  b200_decoder_config cfg{};
  struct Layer {
    b200_decoder_layer s{};
    // wqkv: all projections the mixer takes from h.  wo: W_o, in parallel layers [W_o | W_down] over concatenated columns.
    b200_qweight *wqkv = nullptr, *wo = nullptr, *wgu = nullptr, *wdown = nullptr, *wuk = nullptr, *wuv = nullptr, *we_gu = nullptr, *we_down = nullptr;
    // wuq: queries from their latent.  wgates: gates of the matrix memory, or of the LRU's blocks.
    b200_qweight *wuq = nullptr, *wgates = nullptr, *wrouter = nullptr;
    float *bias = nullptr, *sinks = nullptr, *slopes = nullptr, *norm1 = nullptr, *norm2 = nullptr, *post1 = nullptr, *post2 = nullptr;
    float *dkv_norm = nullptr, *a2 = nullptr, *a2_bias = nullptr, *head_norm = nullptr, *depth = nullptr;
    float *dq_norm = nullptr, *q_norm = nullptr, *k_norm = nullptr, *conv_bias = nullptr, *gate_bias = nullptr, *mem_norm = nullptr;
    float *lru_bias = nullptr, *lru_rate = nullptr;  // [y | x | r | i], [width]
    __nv_bfloat16* conv = nullptr;                   // [taps][channels]
    // of the two sublayers: convolution of what they read, gate on their result
    __nv_bfloat16* in_conv[2] = {};
    b200_qweight* wgate[2] = {};
    float* out_gate_bias[2] = {};
    float *dist = nullptr, *rate = nullptr, *dt_bias = nullptr;  // bias by distance, [heads][dist_len]; of the delta rule, [heads]
    int dist_len = 0, hidden = 0;
    int* table = nullptr;
    std::vector<int> h_table;
    int moe = -1;       // place among the layers with experts
    int rotation = -1;  // its rotation table
    int qkv_n() const {
      if (s.mixer == B200_MIX_LATENT) return (s.q_rank > 0 ? s.q_rank : q_n()) + (s.kv_source > 0 ? 0 : s.kv_rank + s.rot_dim);
      if (s.mixer == B200_MIX_LRU) return 2 * attn_n();
      if (delta()) return b200_delta_channels(s.n_heads, s.n_kv_heads, s.key_dim, s.value_dim) + s.n_heads * (s.value_dim + 2);
      if (s.mixer == B200_MIX_GLA) return 2 * s.n_heads * (s.key_dim + s.value_dim) + s.decay_rank;
      return attention_n() + 2 * s.mem_heads * (s.mem_key_dim + s.mem_value_dim);
    }
    int q_n() const { return s.n_heads * (s.key_dim + s.rot_dim); }  // queries of latent attention
    bool delta() const { return s.mixer == B200_MIX_DELTA; }
    int attention_n() const { return s.n_heads * s.key_dim + (s.kv_source > 0 ? 0 : s.n_kv_heads * (s.key_dim + s.value_dim)); }
    int mem_n() const { return s.mem_heads * s.mem_value_dim; }
    int mem_col() const { return pad64(attn_n()); }
    int router_n() const { return s.flags & B200_DEC_ROUTER ? s.n_experts : 0; }
    // state of a slot: the matrix memory, then the convolution's inputs
    int conv_off() const { return s.mem_heads > 0 ? (b200_memory_elems(s.mem_heads, s.mem_key_dim, s.mem_value_dim) + 3) / 4 * 4 : 0; }
    int mixer_elems() const {
      int n = 0;
      if (delta()) n = (b200_delta_elems(s.n_heads, s.n_kv_heads, s.key_dim, s.value_dim, s.conv_taps) + 3) / 4 * 4;
      if (s.mixer == B200_MIX_GLA) n = s.n_heads * s.key_dim * s.value_dim;
      if (s.mixer == B200_MIX_LRU) n = (b200_lru_elems(attn_n(), s.conv_taps) + 3) / 4 * 4;
      if (s.mixer == B200_MIX_ATTENTION) n = (conv_off() + (s.conv_taps > 1 ? s.conv_taps - 1 : 0) * attention_n() + 3) / 4 * 4;
      return n;
    }
    // behind the mixer's part: inputs of the convolutions in front of the sublayers
    bool second() const { return (s.ffn > 0 || s.n_experts > 0) && !parallel(); }
    int in_conv_off(int which) const { return (mixer_elems() + 3) / 4 * 4 + which * (s.input_taps - 1) * hidden; }
    int state_elems() const {
      if (s.input_taps < 2) return mixer_elems();
      return (in_conv_off(second() ? 2 : 1) + 3) / 4 * 4;
    }
    int lru_group() const { return pad64(s.value_dim); }
    int attn_n() const { return s.n_heads * s.value_dim; }
    bool parallel() const { return (s.flags & B200_DEC_PARALLEL) != 0; }
    bool gelu() const { return (s.flags & B200_DEC_FF_GELU) != 0; }
    bool plain_ff() const { return (s.flags & (B200_DEC_FF_GELU | B200_DEC_FF_RELU2)) != 0; }  // without a gate
    int epilogue() const { return gelu() ? B200_EPI_GELU : (plain_ff() ? B200_EPI_RELU2 : B200_EPI_SWIGLU); }
    SwigluShape swiglu() const { return SwigluShape{s.ff_limit, s.ff_alpha > 0.f ? s.ff_alpha : 1.f, s.ff_shift}; }
    bool shared_gate() const { return (s.flags & B200_DEC_SHARED_GATE) != 0; }
    int ffn_col() const { return mem_col() + (s.mem_heads > 0 ? pad64(mem_n()) : 0); }
    int out_k() const { return ffn_col() + (parallel() && s.ffn > 0 ? pad64(s.ffn) : 0); }  // columns wo reads
    int plain_stride() const { return pad64(s.key_dim); }
    int latent_width() const { return (s.kv_rank + s.rot_dim + 15) / 16 * 16; }
    std::vector<int> projections() const {
      if (s.mixer == B200_MIX_LATENT) {
        std::vector<int> w{s.q_rank > 0 ? B200_DEC_W_DQ : B200_DEC_W_Q};
        if (s.kv_source == 0) w.push_back(B200_DEC_W_DKV);
        return w;
      }
      if (s.mixer == B200_MIX_LRU) return {B200_DEC_W_LRU_Y, B200_DEC_W_LRU_X};
      if (s.mixer == B200_MIX_GLA) return {B200_DEC_W_Q, B200_DEC_W_K, B200_DEC_W_V, B200_DEC_W_OUT_GATE, B200_DEC_W_A1};
      if (delta()) return {B200_DEC_W_Q, B200_DEC_W_K, B200_DEC_W_V, B200_DEC_W_OUT_GATE, B200_DEC_W_BETA, B200_DEC_W_DECAY};
      if (s.kv_source > 0) return {B200_DEC_W_Q};
      std::vector<int> w{B200_DEC_W_Q, B200_DEC_W_K, B200_DEC_W_V};
      if (s.mem_heads > 0) w.insert(w.end(), {B200_DEC_W_MEM_Q, B200_DEC_W_MEM_K, B200_DEC_W_MEM_V, B200_DEC_W_MEM_G});
      return w;
    }
    b200_kv_layer cache() const {
      if (s.mixer == B200_MIX_LATENT && s.kv_source == 0) return b200_kv_layer{1, s.kv_rank + s.rot_dim, s.kv_rank, 1, state_elems()};
      if (s.mixer == B200_MIX_GLA || s.mixer == B200_MIX_LRU || delta() || s.kv_source > 0) return b200_kv_layer{0, 0, 0, 0, state_elems()};
      return b200_kv_layer{s.n_kv_heads, s.key_dim, s.value_dim, 0, state_elems()};
    }
  };
  // Rotations of a step, one table per (base, width, scaling) in the stack.
  struct Rotation {
    double base, factor, original, fast, slow;
    int dims;
    double* freq;
    float2* rows;
    double size() const { return factor > 0 ? 0.1 * std::log(factor) + 1.0 : 1.0; }
  };
  std::vector<Rotation> rotations;
  // Experts by token id: plan buffers of every layer that has them (d_moe: the same on the device), and the rows they work on.
  std::vector<MoeTableLayer> moe;
  MoeTableLayer* d_moe = nullptr;
  std::vector<int> moe_layers;
  int n_tables = 0;  // layers whose experts come from a table
  void *moe_x = nullptr, *moe_act = nullptr, *moe_y = nullptr;
  GlaScratch gla;
  bool has_gla = false;  // some layer works chunk by chunk
  void *q_plain = nullptr, *lat_out = nullptr, *q_latent = nullptr;
  float *lru_gates = nullptr, *moe_wts = nullptr;  // gates in front of their activation; weights of a router's experts
  float4* mem_gates = nullptr;
  float* hist = nullptr;  // [layers + 1][max_rows][hidden]: embedding output and results of the layers
  std::vector<Layer> layers;
  struct Run { int layer; bool opens; };  // opens: the first layer of a pass of the loop
  std::vector<Run> runs;
  std::map<std::pair<int, int>, HostTensor> staged;
  __nv_bfloat16 *embed = nullptr, *pos_embed = nullptr;
  float* final_norm = nullptr;
  b200_qweight *head = nullptr, *loop_in = nullptr;
  // activations: residual and embedding output in f32, operands in the model's type
  float *x = nullptr, *x0 = nullptr, *rec = nullptr;
  void *h = nullptr, *cat = nullptr, *y = nullptr, *q = nullptr, *attn = nullptr, *act = nullptr, *last = nullptr;
  void *hc = nullptr, *gate_y = nullptr;  // h + conv(h); rows of a result's gate where the matmul writes them itself
  float* shared_w = nullptr;              // weight of a token's shared expert
  b200_kv* step_kv = nullptr;             // of the step in flight
  int step_reqs = 0;
  int hp = 0, catp = 0;  // padded widths of h and [x ; x0]
  bool attn_mma = true, recording = false;

  size_t elem() const { return cfg.dtype == B200_DT_F32 ? 4 : 2; }
  bool f32() const { return cfg.dtype == B200_DT_F32; }
  ~b200_decoder() override;
  b200_status check_pool(const b200_kv* kv) const override;
  b200_status run_layers(b200_kv* kv, int n_req, int T, int n_logits, void* stream) override;
  b200_status reserve_logit_rows(int rows) override;
  b200_status matmul(const b200_qweight* w, const void* in, int rows, int defer, MatSrc* src, void* stream);
  b200_status rows_step(RowArgs a, int rows, int next, cudaStream_t s, int run = -1, int which = 0);
  b200_status result_gate(const Layer& l, int which, int rows, MatSrc* src, void* stream);
  const void* in_of(const Layer& l) const { return l.s.input_taps > 0 ? hc : h; }  // what a sublayer's matmuls read
  b200_status attention(b200_kv* kv, int run, int rows, void* stream);
  b200_status mixer(b200_kv* kv, int run, int n_req, int T, void* stream);
  b200_status memory(b200_kv* kv, int run, const MatSrc& src, int n_req, int T, void* stream);
  b200_status lru(b200_kv* kv, int run, const MatSrc& src, int n_req, int T, void* stream);
  b200_status experts(const Layer& l, int T, int tile_rows, void* stream);
  b200_status begin_step(b200_kv* kv, int n_req, int T, int tile_rows, void* stream);
  int moe_tile_rows(int T) const;
  int kv_run(int run) const { return layers[runs[run].layer].s.kv_source > 0 ? layers[runs[run].layer].s.kv_source - 1 : run; }  // whose pages it reads
  bool sum_norm() const { return (cfg.flags & B200_DEC_SUM_NORM) != 0; }
};

b200_decoder::~b200_decoder() {
  void* dev[] = {embed, final_norm, x, x0, rec, h, cat, y, q, attn, act, last, q_plain, lat_out, hist, moe_x, moe_act, moe_y, d_moe, q_latent, lru_gates, moe_wts, mem_gates,
                 pos_embed, hc, gate_y, shared_w};
  for (void* p : dev) if (p) cudaFree(p);
  for (Layer& l : layers) {
    void* lp[] = {l.bias, l.sinks, l.slopes, l.norm1, l.norm2, l.post1, l.post2, l.dkv_norm, l.a2, l.a2_bias, l.head_norm, l.depth, l.table,
                  l.dq_norm, l.q_norm, l.k_norm, l.conv, l.conv_bias, l.gate_bias, l.mem_norm, l.lru_bias, l.lru_rate,
                  l.in_conv[0], l.in_conv[1], l.out_gate_bias[0], l.out_gate_bias[1], l.dist, l.rate, l.dt_bias};
    for (void* p : lp) if (p) cudaFree(p);
    for (b200_qweight* w : {l.wqkv, l.wo, l.wgu, l.wdown, l.wuk, l.wuv, l.we_gu, l.we_down, l.wuq, l.wgates, l.wrouter, l.wgate[0], l.wgate[1]}) b200_qweight_destroy(w);
  }
  for (MoeTableLayer& t : moe) {
    void* tp[] = {t.indices, t.offsets, t.order, t.inv_order, t.n_items, t.items};
    for (void* p : tp) if (p) cudaFree(p);
  }
  for (Rotation& t : rotations) {
    if (t.freq) cudaFree(t.freq);
    if (t.rows) cudaFree(t.rows);
  }
  gla.free();
  b200_qweight_destroy(head);
  b200_qweight_destroy(loop_in);
}

b200_status b200_decoder::check_pool(const b200_kv* kv) const {
  bool ok = kv->layered && kv->cfg.n_layers == (int)runs.size() && kv->dev.elem_bytes == (int)elem();
  for (size_t r = 0; ok && r < runs.size(); ++r) {
    const b200_kv_layer want = layers[runs[r].layer].cache();
    const KvLayerDev& L = kv->lay[r];
    ok = L.heads == want.n_kv_heads && L.key_dim == want.key_dim && L.value_dim == want.value_dim && L.values_in_keys == want.values_in_keys &&
         L.rec_elems == want.state_elems && layers[runs[r].layer].s.n_heads <= kv->cfg.n_q_heads;
  }
  if (!ok) { b200_set_error("decoder: the page pool was built for a different model shape"); return B200_ERR_INVALID_ARGUMENT; }
  return B200_OK;
}

b200_status b200_decoder::reserve_logit_rows(int rows) {
  void* p = nullptr;
  if (cudaMalloc(&p, (size_t)rows * hp * elem()) != cudaSuccess) { b200_set_error("decoder: no memory for %d logit rows", rows); return B200_ERR_CUDA; }
  B200_CUDA_TRY(cudaMemset(p, 0, (size_t)rows * hp * elem()));
  cudaFree(last);
  last = p;
  return B200_OK;
}

// y = in W^T.  src describes where the result is: rows of `y`, or the f32 partial sums of a split K (defer = 1: if K was
// split; 2: always f32).
b200_status b200_decoder::matmul(const b200_qweight* w, const void* in, int rows, int defer, MatSrc* src, void* stream) {
  *src = MatSrc{};
  src->y = y;
  src->y_stride = w->n;
  if (f32()) return b200_qmm_f32(w, (const float*)in, rows, (float*)y, w->n, w->n, B200_EPI_NONE, stream);
  b200_qmm_partials p;
  b200_status st = b200_qmm_deferred(w, in, rows, y, defer, stream, &p);
  if (st == B200_OK && p.pending) { src->ws = p.d_ws; src->splits = p.splits; src->tn = p.tn; src->tts = p.tts; }
  return st;
}

// Gate on the result of a sublayer, from the h it is given.
b200_status b200_decoder::result_gate(const Layer& l, int which, int rows, MatSrc* src, void* stream) {
  const b200_qweight* w = l.wgate[which];
  *src = MatSrc{};
  src->y = gate_y;
  src->y_stride = w->n;
  if (f32()) return b200_qmm_f32(w, (const float*)h, rows, (float*)gate_y, w->n, w->n, B200_EPI_NONE, stream);
  b200_qmm_partials p;
  const b200_status st = b200_qmm_deferred_aside(w, h, rows, gate_y, 1, stream, &p);
  if (st == B200_OK && p.pending) { src->ws = p.d_ws; src->splits = p.splits; src->tn = p.tn; src->tts = p.tts; }
  return st;
}

// decoder_rows_kernel with what run `next` reads (its first norm, or [x ; x0] when it opens a pass; nothing past the end).
// next < 0: a.norm_w is already set, for sublayer `which` of run `run`.  The convolution of what a sublayer reads is done here as well.
b200_status b200_decoder::rows_step(RowArgs a, int rows, int next, cudaStream_t s, int run, int which) {
  a.hidden = cfg.hidden;
  a.eps = cfg.norm_eps;
  a.x = x;
  a.x0 = x0;
  a.h = h;
  a.h_stride = hp;
  if (hist) { a.hist = hist; a.hist_stride = (size_t)max_rows * cfg.hidden; }
  if (sum_norm()) {
    if (a.tokens) a.plain_h = 1;
    else a.norm_x = 1;
    a.x_scale = cfg.residual_scale;
  } else if (next >= 0 && next < (int)runs.size()) {
    if (runs[next].opens) { a.cat = cat; a.cat_stride = catp; }
    else {
      a.norm_w = layers[runs[next].layer].norm1;
      run = next;
      which = 0;
    }
  }
  a.pos = d_pos;
  InputConvArgs ic{};
  if (run >= 0 && layers[runs[run].layer].s.input_taps > 0) {
    const Layer& l = layers[runs[run].layer];
    const KvLayerDev& L = step_kv->lay[run];
    ic.conv.taps = l.s.input_taps; ic.conv.channels = cfg.hidden; ic.conv.w = l.in_conv[which];
    ic.conv.state = step_kv->dev.rec_pool + L.rec_off + l.in_conv_off(which); ic.conv.slot_elems = L.rec_elems;
    if (rows == step_reqs) {  // a token per request
      a.conv = ic.conv; a.hc = hc; a.row_seq = d_row_seq; a.pool_state = step_kv->dev.state; a.max_seqs = step_kv->dev.max_seqs;
    } else {
      ic.h = h; ic.hc = hc; ic.hidden = cfg.hidden; ic.stride = hp; ic.max_seqs = step_kv->dev.max_seqs; ic.pool_state = step_kv->dev.state;
      ic.cu = d_cu; ic.row_to_req = d_row_to_req; ic.row_seq = d_row_seq; ic.pos = d_pos;
    }
  }
  const int vec = cfg.hidden % 4 == 0 ? 4 : 1;
  const bool few = rows < 512 || a.hc;
  const int threads = std::min(few ? 512 : 256, (cfg.hidden / vec + 31) / 32 * 32), nq = (cfg.hidden / vec + threads - 1) / threads;
  const size_t smem = vec == 4 && nq <= 4 ? 0 : sizeof(float) * cfg.hidden;
  auto* kernel = f32() ? (few ? rows_kernel<float, true>(vec, nq) : rows_kernel<float, false>(vec, nq))
                       : (few ? rows_kernel<__nv_bfloat16, true>(vec, nq) : rows_kernel<__nv_bfloat16, false>(vec, nq));
  if (smem > 47 * 1024) B200_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  kernel<<<rows, threads, smem, s>>>(a);
  B200_LAUNCH_CHECK();
  return ic.hc ? launch_input_conv(ic, rows, f32(), s) : B200_OK;
}

b200_status b200_decoder::attention(b200_kv* kv, int run, int rows, void* stream) {
  const Layer& l = layers[runs[run].layer];
  WindowAttnCall c;
  c.layer = kv_run(run);
  c.n_q_heads = l.s.n_heads;
  c.window = l.s.window;
  c.q = q;
  c.q_stride = l.s.n_heads * kv->lay[c.layer].kd;
  c.scale = l.s.scale;
  c.slopes_log2 = l.slopes;
  c.sinks_log2 = l.sinks;
  c.dist_log2 = l.dist;
  c.dist_len = l.dist_len;
  c.out = attn;
  c.out_stride = l.out_k();
  if (l.s.mixer == B200_MIX_LATENT) {
    c.out = lat_out;
    c.out_head_stride = pad64(l.s.kv_rank);
    c.out_stride = l.s.n_heads * c.out_head_stride;
  }
  return b200_window_attn_run(kv, c, d_row_seq, d_row_ctx, rows, attn_mma, stream);
}

// Token tile of the experts' matmuls: the rows an expert gets on average, rounded up.
int b200_decoder::moe_tile_rows(int T) const {
  if (f32()) return 64;
  int rows = 0;
  for (int i : moe_layers) rows = std::max(rows, (T * layers[i].s.top_k + layers[i].s.n_experts - 1) / layers[i].s.n_experts);
  return std::min(128, std::max(16, (rows + 15) / 16 * 16));
}

// What the layers of a step share: attention plans, chunks of the recurrent layers, rotations, experts.
b200_status b200_decoder::begin_step(b200_kv* kv, int n_req, int T, int tile_rows, void* stream) {
  b200_decoder* m = this;
  cudaStream_t cs = (cudaStream_t)stream;
  b200_status st = B200_OK;
  step_kv = kv;
  step_reqs = n_req;
  // one plan per (window, GQA group) of the stack, shared by its layers (latent layers: of the same key width)
  std::vector<std::tuple<int, int, int>> planned;
  for (size_t r = 0; r < runs.size(); ++r) {
    const b200_decoder_layer& s = layers[runs[r].layer].s;
    if (s.mixer == B200_MIX_GLA || s.mixer == B200_MIX_LRU || s.mixer == B200_MIX_DELTA) continue;
    const bool latent = s.mixer == B200_MIX_LATENT;
    const int pages_of = kv_run((int)r);
    const std::tuple<int, int, int> key{s.window, latent ? s.n_heads : s.n_heads / s.n_kv_heads, latent ? kv->lay[pages_of].kd : 0};
    if (!attn_mma || !b200_window_attn_takes_mma(kv, pages_of) || std::find(planned.begin(), planned.end(), key) != planned.end()) continue;
    planned.push_back(key);
    MODEL_STEP_CAT(0, b200_window_attn_plan(kv, pages_of, std::get<0>(key), std::get<1>(key), d_row_seq, d_row_ctx, T, stream));
  }
  if (has_gla && T > n_req) MODEL_STEP_CAT(0, b200_gla_plan(gla, d_cu, n_req, T, stream));
  for (const Rotation& t : rotations) MODEL_STEP(b200_rotation_table(t.freq, t.dims, t.size(), d_pos, T, t.rows, stream));
  if (n_tables > 0) {
    int most = 0;
    for (const MoeTableLayer& t : moe) most = std::max(most, t.n_experts);
    MODEL_STEP(b200_moe_table_plan(d_moe, n_tables, most, d_tokens, T, cfg.vocab, tile_rows, stream));
  }
  return B200_OK;
}

// Mixer of one layer run: h -> the rows W_o reads.
b200_status b200_decoder::mixer(b200_kv* kv, int run, int n_req, int T, void* stream) {
  b200_decoder* m = this;
  cudaStream_t cs = (cudaStream_t)stream;
  const Layer& l = layers[runs[run].layer];
  const b200_decoder_layer& s = l.s;
  b200_status st = B200_OK;
  MatSrc src;
  if (s.mem_heads > 0) {  // the gates' sums stay f32, and are used up before the next product
    MODEL_STEP_CAT(1, matmul(l.wgates, in_of(l), T, 2, &src, stream));
    MemoryGates g;
    g.layer = run; g.heads = s.mem_heads; g.m_off = s.mem_heads * s.mem_key_dim * b200_memory_width(s.mem_value_dim);
    g.src = src; g.bias = l.gate_bias; g.cap = s.mem_gate_cap; g.out = mem_gates;
    MODEL_STEP_CAT(0, b200_memory_gates(kv, g, d_cu, d_row_seq, d_pos, n_req, T, stream));
  }
  MODEL_STEP_CAT(1, matmul(l.wqkv, in_of(l), T, 1, &src, stream));
  if (l.delta()) {
    DeltaCall c;
    c.layer = run; c.heads = s.n_heads; c.kv_heads = s.n_kv_heads; c.dk = s.key_dim; c.dv = s.value_dim; c.src = src;
    c.conv.taps = s.conv_taps; c.conv.w = l.conv; c.rate = l.rate; c.dt_bias = l.dt_bias; c.norm = l.head_norm; c.eps = cfg.norm_eps;
    c.out = attn; c.out_stride = l.out_k();
    MODEL_STEP_CAT(2, b200_delta_prep(kv, gla, c, d_cu, d_row_to_req, d_row_seq, d_pos, T, stream));
    MODEL_STEP_CAT(0, b200_delta_run(kv, gla, c, d_cu, d_row_seq, d_pos, n_req, T, attn_mma, stream));
    return B200_OK;
  }
  if (s.mixer == B200_MIX_LRU) return lru(kv, run, src, n_req, T, stream);
  if (s.mixer == B200_MIX_GLA) {
    GlaCall c;
    c.layer = run; c.heads = s.n_heads; c.dk = s.key_dim; c.dv = s.value_dim; c.rank = s.decay_rank; c.src = src;
    c.a2 = l.a2; c.a2_bias = l.a2_bias; c.norm = l.head_norm; c.eps = cfg.norm_eps;
    c.q_scale = (float)(1.0 / std::sqrt((double)s.key_dim));
    c.inv_tau = 1.0f / s.decay_tau;
    c.out = attn; c.out_stride = l.out_k();
    MODEL_STEP_CAT(0, b200_gla_run(kv, gla, c, d_cu, d_row_seq, d_pos, n_req, T, attn_mma, stream));
    return B200_OK;
  }
  if (s.mixer == B200_MIX_LATENT) {
    const int pages_of = kv_run(run);
    LatentPrep p;
    p.layer = pages_of; p.heads = s.n_heads; p.dim = s.key_dim; p.rot = s.rot_dim; p.rank = s.kv_rank; p.src = src; p.norm = l.dkv_norm;
    p.halves = (s.flags & B200_DEC_ROT_HALVES) != 0; p.keys = s.kv_source == 0;
    p.eps = cfg.norm_eps; p.rotation = l.rotation >= 0 ? rotations[l.rotation].rows : nullptr;
    p.q_plain = q_plain; p.plain_stride = l.plain_stride(); p.q = q;
    if (s.q_rank > 0) {
      p.heads = 0; p.q_rank = s.q_rank; p.q_norm = l.dq_norm; p.q_latent = q_latent; p.q_latent_stride = pad64(s.q_rank);
      MODEL_STEP_CAT(2, b200_latent_prep(kv, p, d_pos, d_row_seq, T, stream));
      MODEL_STEP_CAT(1, matmul(l.wuq, q_latent, T, 1, &src, stream));
      p.heads = s.n_heads; p.q_rank = 0; p.q_latent_stride = 0; p.src = src; p.keys = false;
    }
    MODEL_STEP_CAT(2, b200_latent_prep(kv, p, d_pos, d_row_seq, T, stream));
    const int H = s.n_heads, kd = kv->lay[pages_of].kd, lat = pad64(s.kv_rank);
    auto blocks = [&](const b200_qweight* w, const void* in, int in_group, void* out, int out_stride, int out_group) {
      return f32() ? b200_qmm_f32_blocks(w, (const float*)in, H * in_group, in_group, T, (float*)out, out_stride, out_group, stream)
                   : b200_qmm_blocks(w, in, H * in_group, in_group, T, out, out_stride, out_group, stream);
    };
    MODEL_STEP_CAT(1, blocks(l.wuk, q_plain, l.plain_stride(), q, H * kd, kd));
    MODEL_STEP_CAT(0, attention(kv, run, T, stream));
    MODEL_STEP_CAT(1, blocks(l.wuv, lat_out, lat, attn, l.out_k(), s.value_dim));
    return B200_OK;
  }
  QkvArgs a;
  a.d = kv->dev; a.L = kv->lay[kv_run(run)]; a.src = src; a.bias = l.bias; a.hq = s.n_heads; a.qk_norm = s.flags & B200_DEC_QK_NORM ? 1 : 0;
  a.norm_row = (s.flags & B200_DEC_QK_NORM_ROW) != 0; a.keys = s.kv_source == 0; a.temp_coef = s.q_temp_coef; a.temp_every = s.q_temp_every;
  a.eps = cfg.norm_eps; a.q = q; a.q_stride = s.n_heads * a.L.kd; a.pos = d_pos; a.row_seq = d_row_seq;
  a.cu = d_cu; a.row_to_req = d_row_to_req; a.q_norm = l.q_norm; a.k_norm = l.k_norm;
  if (l.rotation >= 0) { a.rotation = rotations[l.rotation].rows; a.rot = s.rot_dim; a.halves = s.flags & B200_DEC_ROT_HALVES ? 1 : 0; }
  if (s.conv_taps > 0) {
    a.conv.taps = s.conv_taps; a.conv.channels = l.attention_n(); a.conv.w = l.conv;
    a.conv.state = kv->dev.rec_pool + kv->lay[run].rec_off + l.conv_off(); a.conv.slot_elems = kv->lay[run].rec_elems;
  }
  if (s.mem_heads > 0) a.v_scale = s.mix_scale;  // the factor of the whole mixer
  MODEL_STEP_CAT(2, launch_qkv(a, T, cs));
  if (s.mem_heads > 0 && (st = memory(kv, run, src, n_req, T, stream)) != B200_OK) return st;
  MODEL_STEP_CAT(0, attention(kv, run, T, stream));
  return B200_OK;
}

// The matrix memory beside attention: its part of the projection -> its columns of the rows W_o reads.
b200_status b200_decoder::memory(b200_kv* kv, int run, const MatSrc& src, int n_req, int T, void* stream) {
  b200_decoder* m = this;
  cudaStream_t cs = (cudaStream_t)stream;
  const Layer& l = layers[runs[run].layer];
  const b200_decoder_layer& s = l.s;
  b200_status st = B200_OK;
  GlaCall c;
  c.layer = run; c.heads = s.mem_heads; c.dk = s.mem_key_dim; c.dv = s.mem_value_dim; c.src = src; c.col0 = l.attention_n();
  c.gates = mem_gates; c.norm = l.mem_norm; c.eps = cfg.norm_eps; c.den_eps = kMemoryEps; c.out_scale = s.mem_scale;
  c.q_scale = (float)(1.0 / std::sqrt((double)s.mem_key_dim));
  c.out = (char*)attn + l.mem_col() * elem(); c.out_stride = l.out_k();
  MODEL_STEP_CAT(0, b200_gla_run(kv, gla, c, d_cu, d_row_seq, d_pos, n_req, T, attn_mma, stream));
  return B200_OK;
}

b200_status b200_decoder::lru(b200_kv* kv, int run, const MatSrc& src, int n_req, int T, void* stream) {
  b200_decoder* m = this;
  cudaStream_t cs = (cudaStream_t)stream;
  const Layer& l = layers[runs[run].layer];
  const b200_decoder_layer& s = l.s;
  b200_status st = B200_OK;
  const int W = l.attn_n(), ub = l.lru_group();
  LruCall c;
  c.layer = run; c.width = W; c.blocks = s.n_heads; c.src = src; c.y_bias = l.lru_bias; c.x_bias = l.lru_bias + W;
  c.conv.taps = s.conv_taps; c.conv.w = l.conv; c.conv.bias = l.conv_bias; c.u = q_plain; c.u_group = ub; c.gates = lru_gates;
  c.r_bias = l.lru_bias + 2 * W; c.i_bias = l.lru_bias + 3 * W; c.rate = l.lru_rate; c.out = attn; c.out_stride = l.out_k();
  MODEL_STEP_CAT(2, b200_lru_prep(kv, c, d_cu, d_row_to_req, d_row_seq, d_pos, T, stream));
  MODEL_STEP_CAT(1, f32() ? b200_qmm_f32_blocks(l.wgates, (const float*)q_plain, s.n_heads * ub, ub, T, lru_gates, 2 * W, 2 * s.value_dim, stream)
                          : b200_qmm_blocks(l.wgates, q_plain, s.n_heads * ub, ub, T, lru_gates, 2 * W, 2 * s.value_dim, stream, true));
  MODEL_STEP_CAT(0, b200_lru_scan(kv, c, d_cu, d_row_seq, d_pos, n_req, T, stream));
  return B200_OK;
}

// The experts of one layer: h -> moe_y, one row per assignment in the experts' order.
b200_status b200_decoder::experts(const Layer& l, int T, int tile_rows, void* stream) {
  b200_decoder* m = this;
  cudaStream_t cs = (cudaStream_t)stream;
  b200_status st = B200_OK;
  const MoeTableLayer& t = moe[l.moe];
  const void* in = in_of(l);
  const int A = T * t.top, act_w = pad64(l.s.expert_ffn), items = std::min(A, t.n_experts + A / tile_rows);
  if (l.wrouter) {
    MatSrc z;
    MODEL_STEP_CAT(1, matmul(l.wrouter, in, T, 2, &z, stream));
    RouterScores scores;
    if (l.s.flags & B200_DEC_ROUTER_PLAIN) { scores.renormalise = false; scores.scale = l.s.router_scale; }
    if (l.shared_gate()) scores.shared = shared_w;
    MODEL_STEP(b200_moe_route_plan(t, z, f32(), std::max(l.s.n_groups, 1), l.s.n_groups > 0 ? l.s.keep_groups : 1, T, tile_rows, moe_wts, stream, scores));
  }
  if (f32()) {
    MODEL_STEP_CAT(1, b200_qmm_f32_grouped(l.we_gu, (const float*)in, t.order, t.top, (float*)moe_act, act_w, l.epilogue(), t.items, t.n_items, items, stream));
    MODEL_STEP_CAT(1, b200_qmm_f32_grouped(l.we_down, (const float*)moe_act, nullptr, 1, (float*)moe_y, hp, B200_EPI_NONE, t.items, t.n_items, items, stream));
    return B200_OK;
  }
  MODEL_STEP(b200_moe_gather_order(in, t.order, t.top, A, hp, moe_x, stream));
  MODEL_STEP_CAT(1, b200_qmm_grouped(l.we_gu, moe_x, A, moe_act, l.epilogue(), nullptr, 0.f, t.items, t.n_items, items, tile_rows, stream));
  MODEL_STEP_CAT(1, b200_qmm_grouped(l.we_down, moe_act, A, moe_y, B200_EPI_NONE, nullptr, 0.f, t.items, t.n_items, items, tile_rows, stream));
  return B200_OK;
}

b200_status b200_decoder::run_layers(b200_kv* kv, int n_req, int T, int n_logits, void* stream) {
  b200_decoder* m = this;
  cudaStream_t cs = (cudaStream_t)stream;
  b200_status st = B200_OK;
  MatSrc src;
  const int tile_rows = moe_tile_rows(T);
  if ((st = begin_step(kv, n_req, T, tile_rows, stream)) != B200_OK) return st;
  {
    RowArgs a{};
    a.tokens = d_tokens;
    a.embed = embed;
    a.vocab = cfg.vocab;
    a.embed_scale = cfg.embed_scale;
    a.pos_embed = pos_embed;
    a.max_positions = max_positions;
    MODEL_STEP(rows_step(a, T, 0, cs));
  }
  for (size_t r = 0; r < runs.size(); ++r) {
    const Layer& l = layers[runs[r].layer];
    const b200_decoder_layer& s = l.s;
    if (runs[r].opens) {  // x = W_in [x ; x0]; the residual is f32, so the product stays f32
      MODEL_STEP_CAT(1, matmul(loop_in, cat, T, 2, &src, stream));
      RowArgs a{};
      a.src = src;
      a.replace = 1;
      a.norm_w = l.norm1;
      MODEL_STEP(rows_step(a, T, -1, cs, (int)r, 0));
    }
    MatSrc gate;
    const bool gated = (s.flags & B200_DEC_RESULT_GATE) != 0;
    // SwiGLU of the dense feed-forward, experts: both from h
    auto feed_forward = [&](void* out, int out_stride) -> b200_status {
      if (s.n_experts > 0 && (st = experts(l, T, tile_rows, stream)) != B200_OK) return st;
      if (s.ffn == 0) return B200_OK;
      if (f32()) MODEL_STEP_CAT(1, b200_qmm_f32_shaped(l.wgu, (const float*)in_of(l), T, (float*)out, out_stride, pad64(s.ffn), l.epilogue(), stream, l.swiglu()));
      else MODEL_STEP_CAT(1, b200_qmm_to(l.wgu, in_of(l), T, out, out_stride, l.epilogue(), stream, l.swiglu()));
      return B200_OK;
    };
    auto last_rows = [&](const float* post) -> b200_status {  // the layer's last sublayer joins the residual
      RowArgs a{};
      if (sum_norm()) a.norm_w = s.ffn > 0 || s.n_experts > 0 ? l.norm2 : l.norm1;
      a.src = src;
      a.post_w = post;
      if (s.n_experts > 0) {
        a.moe_y = moe_y; a.moe_rows = moe[l.moe].inv_order; a.moe_k = s.top_k; a.moe_stride = hp; a.moe_w = 1.0f / (float)s.top_k;
        if (l.wrouter) a.moe_wts = moe_wts;
        if (l.shared_gate()) a.src_scale = shared_w;
      }
      if (gated) { a.gate = gate; a.gate_bias = l.out_gate_bias[l.second() ? 1 : 0]; }
      if (l.depth) { a.depth = l.depth; a.n_hist = (int)r + 1; }
      return rows_step(a, T, (int)r + 1, cs);
    };
    if (l.parallel()) {
      if ((st = feed_forward((char*)attn + l.ffn_col() * elem(), l.out_k())) != B200_OK) return st;
      if ((st = mixer(kv, (int)r, n_req, T, stream)) != B200_OK) return st;
      MODEL_STEP_CAT(1, matmul(l.wo, attn, T, 1, &src, stream));
      MODEL_STEP(last_rows(nullptr));
    } else {
      const bool ff = s.ffn > 0 || s.n_experts > 0;
      if (gated) MODEL_STEP_CAT(1, result_gate(l, 0, T, &gate, stream));
      if ((st = mixer(kv, (int)r, n_req, T, stream)) != B200_OK) return st;
      MODEL_STEP_CAT(1, matmul(l.wo, attn, T, 1, &src, stream));
      if (!ff) {
        MODEL_STEP(last_rows(l.post1));
      } else {
        RowArgs a{};
        a.src = src;
        a.post_w = l.post1;
        a.norm_w = sum_norm() ? l.norm1 : l.norm2;
        if (gated) { a.gate = gate; a.gate_bias = l.out_gate_bias[0]; }
        MODEL_STEP(rows_step(a, T, -1, cs, (int)r, 1));
        if (gated) MODEL_STEP_CAT(1, result_gate(l, 1, T, &gate, stream));
        if ((st = feed_forward(act, pad64(s.ffn))) != B200_OK) return st;
        src = MatSrc{};
        if (s.ffn > 0) MODEL_STEP_CAT(1, matmul(l.wdown, act, T, 1, &src, stream));
        MODEL_STEP(last_rows(l.post2));
      }
    }
    if (recording)
      B200_CUDA_TRY(cudaMemcpyAsync(rec + r * (size_t)max_rows * cfg.hidden, x, sizeof(float) * (size_t)T * cfg.hidden, cudaMemcpyDeviceToDevice, cs));
  }
  auto head_rows = [&]() -> b200_status {
    if (f32()) decoder_final_kernel<float><<<n_logits, 256, 0, cs>>>(x, d_logit_row, final_norm, (float*)last, cfg.hidden, hp, cfg.norm_eps);
    else decoder_final_kernel<__nv_bfloat16><<<n_logits, 256, 0, cs>>>(x, d_logit_row, final_norm, (__nv_bfloat16*)last, cfg.hidden, hp, cfg.norm_eps);
    B200_LAUNCH_CHECK();
    return B200_OK;
  };
  MODEL_STEP(head_rows());
  if (f32()) {
    MODEL_STEP_CAT(1, b200_qmm_f32(head, (const float*)last, n_logits, (float*)logits, cfg.vocab, cfg.vocab, B200_EPI_NONE, stream));
    return B200_OK;
  }
  MODEL_STEP_CAT(1, matmul(head, last, n_logits, 2, &src, stream));
  auto finish = [&]() -> b200_status {
    decoder_logits_kernel<<<dim3((cfg.vocab + 255) / 256, n_logits), 256, 0, cs>>>(src, (float*)logits, cfg.vocab);
    B200_LAUNCH_CHECK();
    return B200_OK;
  };
  MODEL_STEP(finish());
  return B200_OK;
}

// ---- construction and weights -----------------------------------------------------------------------------------
namespace {

// Elements of one tensor of the configuration; 0 when the layer does not have it.
uint64_t tensor_elems(const b200_decoder* m, int layer, int which) {
  const b200_decoder_config& c = m->cfg;
  const uint64_t D = c.hidden;
  switch (which) {
    case B200_DEC_W_HEAD: case B200_DEC_W_EMBED: return (uint64_t)c.vocab * D;
    case B200_DEC_W_POS: return (uint64_t)c.max_positions * D;
    case B200_DEC_W_LOOP_IN: return c.loop_times > 0 ? 2 * D * D : 0;
    case B200_DEC_FINAL_NORM: return c.flags & B200_DEC_SCALAR_NORM ? 1 : D;
    default: break;
  }
  const b200_decoder_layer& s = m->layers[layer].s;
  const uint64_t H = s.n_heads, norm = c.flags & B200_DEC_SCALAR_NORM ? 1 : D, ef = (uint64_t)s.n_experts * s.expert_ffn;
  const bool latent = s.mixer == B200_MIX_LATENT, gla = s.mixer == B200_MIX_GLA, soft = s.mixer == B200_MIX_ATTENTION, lru = s.mixer == B200_MIX_LRU,
             delta = s.mixer == B200_MIX_DELTA, own = !soft || s.kv_source == 0;
  const uint64_t MH = s.mem_heads, mk = MH * s.mem_key_dim, mv = MH * s.mem_value_dim, W = lru ? H * s.value_dim : 0;
  const uint64_t gate = m->layers[layer].plain_ff() ? 0 : 1, taps = soft || delta ? s.conv_taps : 0, weighed = soft && s.flags & B200_DEC_QK_NORM_WEIGHT ? s.key_dim : 0;
  const uint64_t qn = (delta ? s.n_kv_heads : H) * (s.key_dim + (latent ? s.rot_dim : 0)), kn = own ? (gla ? H : s.n_kv_heads) * (uint64_t)s.key_dim : 0,
                 vn = own ? (gla || delta ? H : s.n_kv_heads) * (uint64_t)s.value_dim : 0;
  const bool norm_row = soft && s.flags & B200_DEC_QK_NORM_ROW, result_gate = s.flags & B200_DEC_RESULT_GATE;
  const bool bias = soft && s.flags & B200_DEC_QKV_BIAS, post = s.flags & B200_DEC_POST_NORM;
  const bool ff = s.ffn > 0 || s.n_experts > 0, second = ff && !(s.flags & B200_DEC_PARALLEL);
  switch (which) {
    case B200_DEC_W_Q: return lru ? 0 : qn * (latent && s.q_rank > 0 ? s.q_rank : D);
    case B200_DEC_W_K: return latent || lru ? 0 : kn * D;
    case B200_DEC_W_V: return latent || lru ? 0 : vn * D;
    case B200_DEC_W_O: return D * H * s.value_dim;
    case B200_DEC_W_GATE: return gate * D * s.ffn;
    case B200_DEC_W_UP: case B200_DEC_W_DOWN: return D * s.ffn;
    case B200_DEC_B_Q: return bias ? qn : 0;
    case B200_DEC_B_K: return bias ? kn : 0;
    case B200_DEC_B_V: return bias ? vn : 0;
    case B200_DEC_W_SINK: return s.flags & B200_DEC_SINK ? H : 0;
    case B200_DEC_NORM1: return norm;
    case B200_DEC_NORM2: return second ? norm : 0;
    case B200_DEC_POSTNORM1: return post ? norm : 0;
    case B200_DEC_POSTNORM2: return post && second ? norm : 0;
    case B200_DEC_W_DKV: return latent && s.kv_source == 0 ? (uint64_t)(s.kv_rank + s.rot_dim) * D : 0;
    case B200_DEC_DKV_NORM: return latent && s.kv_source == 0 ? s.kv_rank : 0;
    case B200_DEC_W_DQ: return latent ? s.q_rank * D : 0;
    case B200_DEC_DQ_NORM: return latent ? s.q_rank : 0;
    case B200_DEC_W_UK: return latent ? H * s.key_dim * s.kv_rank : 0;
    case B200_DEC_W_UV: return latent ? H * s.value_dim * s.kv_rank : 0;
    case B200_DEC_W_OUT_GATE: return gla || delta ? vn * D : 0;
    case B200_DEC_W_A1: return gla ? s.decay_rank * D : 0;
    case B200_DEC_W_A2: return gla ? kn * s.decay_rank : 0;
    case B200_DEC_B_A2: return gla ? kn : 0;
    case B200_DEC_HEAD_NORM: return gla || delta ? s.value_dim : 0;
    case B200_DEC_W_EXPERT_GATE: return gate * ef * D;
    case B200_DEC_W_EXPERT_UP: case B200_DEC_W_EXPERT_DOWN: return ef * D;
    case B200_DEC_Q_NORM: return norm_row ? qn : weighed;
    case B200_DEC_K_NORM: return norm_row ? kn : weighed;
    case B200_DEC_CONV_Q: return qn * taps;
    case B200_DEC_CONV_K: return kn * taps;
    case B200_DEC_CONV_V: return vn * taps;
    case B200_DEC_W_MEM_Q: case B200_DEC_W_MEM_K: return mk * D;
    case B200_DEC_W_MEM_V: case B200_DEC_W_MEM_G: case B200_DEC_W_MEM_O: return mv * D;
    case B200_DEC_W_MEM_I: case B200_DEC_W_MEM_F: return MH * D;
    case B200_DEC_B_MEM_I: case B200_DEC_B_MEM_F: return MH;
    case B200_DEC_MEM_NORM: return mv;
    case B200_DEC_W_LRU_Y: case B200_DEC_W_LRU_X: return W * D;
    case B200_DEC_W_LRU_R: case B200_DEC_W_LRU_I: return W * s.value_dim;
    case B200_DEC_LRU_CONV: return W * s.conv_taps;
    case B200_DEC_B_LRU_Y: case B200_DEC_B_LRU_X: case B200_DEC_B_LRU_CONV: case B200_DEC_B_LRU_R: case B200_DEC_B_LRU_I: case B200_DEC_LRU_LAMBDA: return W;
    case B200_DEC_W_ROUTER: return s.flags & B200_DEC_ROUTER ? (uint64_t)s.n_experts * D : 0;
    case B200_DEC_W_REL: return soft ? (uint64_t)s.rel_buckets * H : 0;
    case B200_DEC_IN_CONV1: return D * s.input_taps;
    case B200_DEC_IN_CONV2: return second ? D * s.input_taps : 0;
    case B200_DEC_W_RESULT_GATE1: return result_gate ? D * D : 0;
    case B200_DEC_W_RESULT_GATE2: return result_gate && second ? D * D : 0;
    case B200_DEC_B_RESULT_GATE1: return result_gate ? D : 0;
    case B200_DEC_B_RESULT_GATE2: return result_gate && second ? D : 0;
    case B200_DEC_W_BETA: case B200_DEC_W_DECAY: return delta ? H * D : 0;
    case B200_DEC_A_LOG: case B200_DEC_DT_BIAS: return delta ? H : 0;
    case B200_DEC_W_SHARED_GATE: return s.flags & B200_DEC_SHARED_GATE ? D : 0;
    case B200_DEC_DEPTH: return c.flags & B200_DEC_DEPTH_AVERAGE ? layer + 2 : 0;
    default: return 0;
  }
}

bool global_tensor(int which) {
  return which == B200_DEC_W_HEAD || which == B200_DEC_W_EMBED || which == B200_DEC_W_POS || which == B200_DEC_W_LOOP_IN || which == B200_DEC_FINAL_NORM;
}

b200_status take(b200_decoder* m, int layer, int which, std::vector<uint16_t>* out) {
  auto it = m->staged.find({global_tensor(which) ? -1 : layer, which});
  if (it == m->staged.end()) { b200_set_error("decoder: the %s tensor of layer %d was never set", kTensorNames[which], layer); return B200_ERR_INVALID_ARGUMENT; }
  *out = std::move(it->second.bits);
  m->staged.erase(it);
  return B200_OK;
}

b200_status upload_f32(const std::vector<float>& v, float** out) {
  B200_CUDA_TRY(cudaMalloc((void**)out, sizeof(float) * std::max<size_t>(v.size(), 1)));
  B200_CUDA_TRY(cudaMemcpy(*out, v.data(), sizeof(float) * v.size(), cudaMemcpyHostToDevice));
  return B200_OK;
}

b200_status take_vector(b200_decoder* m, int layer, int which, float** out, double factor = 1.0) {
  std::vector<uint16_t> bits;
  b200_status st = take(m, layer, which, &bits);
  if (st != B200_OK) return st;
  std::vector<float> v(bits.size());
  for (size_t i = 0; i < bits.size(); ++i) v[i] = factor == 1.0 ? bf16_to_f(bits[i]) : (float)(bf16_to_f(bits[i]) * factor);
  return upload_f32(v, out);
}

// A norm's weight over the whole width, also where the checkpoint holds one number.
b200_status take_norm(b200_decoder* m, int layer, int which, float** out, double factor = 1.0) {
  std::vector<uint16_t> bits;
  b200_status st = take(m, layer, which, &bits);
  if (st != B200_OK) return st;
  std::vector<float> v(m->cfg.hidden);
  const float stored_at = m->cfg.flags & B200_DEC_NORM_OFFSET ? 1.f : 0.f;
  for (size_t i = 0; i < v.size(); ++i) v[i] = (float)((stored_at + bf16_to_f(bits[bits.size() == 1 ? 0 : i])) * factor);
  return upload_f32(v, out);
}

// Several vectors one behind the other.
b200_status take_vectors(b200_decoder* m, int layer, std::vector<int> which, float** out) {
  std::vector<float> all;
  for (int w : which) {
    std::vector<uint16_t> bits;
    b200_status st = take(m, layer, w, &bits);
    if (st != B200_OK) return st;
    for (uint16_t b : bits) all.push_back(bf16_to_f(b));
  }
  return upload_f32(all, out);
}

b200_status upload_bf16(const std::vector<uint16_t>& v, __nv_bfloat16** out) {
  B200_CUDA_TRY(cudaMalloc((void**)out, 2 * std::max<size_t>(v.size(), 1)));
  B200_CUDA_TRY(cudaMemcpy(*out, v.data(), 2 * v.size(), cudaMemcpyHostToDevice));
  return B200_OK;
}

// Convolutions [channels, taps] one behind the other, as [taps][channels].
b200_status take_conv(b200_decoder* m, int layer, std::vector<int> which, int taps, __nv_bfloat16** out) {
  std::vector<uint16_t> all;
  for (int w : which) {
    std::vector<uint16_t> bits;
    b200_status st = take(m, layer, w, &bits);
    if (st != B200_OK) return st;
    all.insert(all.end(), bits.begin(), bits.end());
  }
  const size_t channels = all.size() / taps;
  std::vector<uint16_t> t(all.size());
  for (size_t c = 0; c < channels; ++c)
    for (int k = 0; k < taps; ++k) t[k * channels + c] = all[c * taps + k];
  return upload_bf16(t, out);
}

// The blocks' gate matrices, r rows then i rows, and exp's factor lru_decay * softplus(lam).
b200_status take_lru(b200_decoder* m, int layer, b200_decoder::Layer& l) {
  const int n = l.s.n_heads, w = l.s.value_dim, kp = pad64(w);
  std::vector<uint16_t> part[2], lam;
  b200_status st;
  if ((st = take(m, layer, B200_DEC_W_LRU_R, &part[0])) != B200_OK || (st = take(m, layer, B200_DEC_W_LRU_I, &part[1])) != B200_OK ||
      (st = take(m, layer, B200_DEC_LRU_LAMBDA, &lam)) != B200_OK)
    return st;
  std::vector<uint16_t> all((size_t)n * 2 * w * kp, 0);
  for (int b = 0; b < n; ++b)
    for (int g = 0; g < 2; ++g)
      for (int r = 0; r < w; ++r) std::memcpy(&all[((size_t)b * 2 * w + g * w + r) * kp], &part[g][((size_t)b * w + r) * w], sizeof(uint16_t) * w);
  if ((st = b200_qweight_create(B200_Q_BF16, n, 2 * w, kp, all.data(), nullptr, nullptr, &l.wgates)) != B200_OK) return st;
  std::vector<float> rate(lam.size());
  for (size_t i = 0; i < rate.size(); ++i) {
    const double x = bf16_to_f(lam[i]);
    rate[i] = (float)(l.s.lru_decay * (std::max(x, 0.0) + std::log1p(std::exp(-std::fabs(x)))));
  }
  return upload_f32(rate, &l.lru_rate);
}

// Matrices [n, k_i] beside one another as one weight, each padded to a multiple of 64 columns.
b200_status take_beside(b200_decoder* m, int layer, std::vector<std::pair<int, int>> which_k, int n, b200_qweight** out) {
  int kp = 0;
  for (auto& wk : which_k) kp += pad64(wk.second);
  const int np = pad64(n);
  std::vector<uint16_t> w((size_t)np * kp, 0);
  int col = 0;
  for (auto& wk : which_k) {
    std::vector<uint16_t> part;
    b200_status st = take(m, layer, wk.first, &part);
    if (st != B200_OK) return st;
    for (int r = 0; r < n; ++r) std::memcpy(&w[(size_t)r * kp + col], &part[(size_t)r * wk.second], sizeof(uint16_t) * wk.second);
    col += pad64(wk.second);
  }
  return b200_qweight_create(B200_Q_BF16, 1, np, kp, w.data(), nullptr, nullptr, out);
}

// A stack of `count` matrices [n, k] held as [count][n][k] (transposed: [count][k][n]); n rows each, columns padded to 64.
b200_status take_stack(b200_decoder* m, int layer, int which, int count, int n, int k, bool transposed, b200_qweight** out) {
  std::vector<uint16_t> part;
  b200_status st = take(m, layer, which, &part);
  if (st != B200_OK) return st;
  const int kp = pad64(k);
  std::vector<uint16_t> w((size_t)count * n * kp, 0);
  for (int e = 0; e < count; ++e)
    for (int r = 0; r < n; ++r)
      for (int c = 0; c < k; ++c)
        w[((size_t)e * n + r) * kp + c] = part[transposed ? ((size_t)e * k + c) * n + r : ((size_t)e * n + r) * k + c];
  return b200_qweight_create(B200_Q_BF16, count, n, kp, w.data(), nullptr, nullptr, out);
}

// Experts: gate and up rows interleaved, [2 pad(ff), pad(hidden)] (without a gate [pad(ff), pad(hidden)]); down [pad(hidden), pad(ff)].
b200_status take_experts(b200_decoder* m, int layer, b200_decoder::Layer& l) {
  const int E = l.s.n_experts, f = l.s.expert_ffn, D = m->cfg.hidden, fp = pad64(f), dp = pad64(D), per = l.plain_ff() ? 1 : 2;
  std::vector<uint16_t> gate, up, down;
  b200_status st;
  if ((per == 2 && (st = take(m, layer, B200_DEC_W_EXPERT_GATE, &gate)) != B200_OK) || (st = take(m, layer, B200_DEC_W_EXPERT_UP, &up)) != B200_OK ||
      (st = take(m, layer, B200_DEC_W_EXPERT_DOWN, &down)) != B200_OK)
    return st;
  std::vector<uint16_t> w((size_t)E * per * fp * dp, 0);
  for (int e = 0; e < E; ++e)
    for (int r = 0; r < f; ++r) {
      uint16_t* dst = &w[((size_t)e * per * fp + per * r) * dp];
      if (per == 2) std::memcpy(dst, &gate[((size_t)e * f + r) * D], sizeof(uint16_t) * D);
      std::memcpy(dst + (per - 1) * dp, &up[((size_t)e * f + r) * D], sizeof(uint16_t) * D);
    }
  if ((st = b200_qweight_create(B200_Q_BF16, E, per * fp, dp, w.data(), nullptr, nullptr, &l.we_gu)) != B200_OK) return st;
  w.assign((size_t)E * dp * fp, 0);
  for (int e = 0; e < E; ++e)
    for (int r = 0; r < D; ++r) std::memcpy(&w[((size_t)e * dp + r) * fp], &down[((size_t)e * D + r) * f], sizeof(uint16_t) * f);
  return b200_qweight_create(B200_Q_BF16, E, dp, fp, w.data(), nullptr, nullptr, &l.we_down);
}

b200_status upload_table(b200_decoder* m, int layer, b200_decoder::Layer& l) {
  if (l.h_table.empty()) { b200_set_error("decoder: the expert table of layer %d was never set", layer); return B200_ERR_INVALID_ARGUMENT; }
  B200_CUDA_TRY(cudaMalloc((void**)&l.table, sizeof(int) * l.h_table.size()));
  B200_CUDA_TRY(cudaMemcpy(l.table, l.h_table.data(), sizeof(int) * l.h_table.size(), cudaMemcpyHostToDevice));
  m->moe[l.moe].table = l.table;
  return B200_OK;
}

// After the last table is in place: the plan structures the kernels read.
b200_status upload_moe(b200_decoder* m) {
  std::vector<MoeTableLayer> with_table;
  for (const MoeTableLayer& t : m->moe) if (t.table) with_table.push_back(t);
  m->n_tables = (int)with_table.size();
  if (with_table.empty()) return B200_OK;
  if (!m->d_moe) B200_CUDA_TRY(cudaMalloc((void**)&m->d_moe, sizeof(MoeTableLayer) * with_table.size()));
  B200_CUDA_TRY(cudaMemcpy(m->d_moe, with_table.data(), sizeof(MoeTableLayer) * with_table.size(), cudaMemcpyHostToDevice));
  return B200_OK;
}

// Rows of several [n_i, k] matrices, one behind the other or interleaved, as one weight padded to multiples of 64.
b200_status make_weight(const std::vector<const std::vector<uint16_t>*>& parts, int k, bool interleave, b200_qweight** out) {
  size_t n = 0;
  for (auto* p : parts) n += p->size() / k;
  const int np = interleave ? 2 * pad64((int)n / 2) : pad64((int)n), kp = pad64(k);
  std::vector<uint16_t> w((size_t)np * kp, 0);
  size_t row = 0;
  auto put = [&](const std::vector<uint16_t>* p, size_t r) { std::memcpy(&w[row++ * kp], &(*p)[r * k], sizeof(uint16_t) * k); };
  if (interleave) {
    for (size_t r = 0; r < parts[0]->size() / k; ++r) for (auto* p : parts) put(p, r);
  } else {
    for (auto* p : parts) for (size_t r = 0; r < p->size() / k; ++r) put(p, r);
  }
  return b200_qweight_create(B200_Q_BF16, 1, np, kp, w.data(), nullptr, nullptr, out);
}

b200_status take_weight(b200_decoder* m, int layer, std::vector<int> which, int k, bool interleave, b200_qweight** out) {
  std::vector<std::vector<uint16_t>> host(which.size());
  std::vector<const std::vector<uint16_t>*> parts;
  for (size_t i = 0; i < which.size(); ++i) {
    b200_status st = take(m, layer, which[i], &host[i]);
    if (st != B200_OK) return st;
    parts.push_back(&host[i]);
  }
  return make_weight(parts, k, interleave, out);
}

b200_status make_slopes(b200_decoder::Layer& l) {
  if (!(l.s.flags & B200_DEC_DISTANCE_BIAS)) return B200_OK;
  std::vector<float> v(l.s.n_heads);
  for (int h = 0; h < l.s.n_heads; ++h) v[h] = (float)(std::exp2(-8.0 * (h + 1) / l.s.n_heads) * kLog2e);
  return upload_f32(v, &l.slopes);
}

// The rows of a distance table [buckets][heads] spread out over distances: one row each for the near half, the far half by the logarithm, up
// to the first distance of the last row.
b200_status make_distances(b200_decoder::Layer& l, const std::vector<float>& table) {
  const int B = l.s.rel_buckets, H = l.s.n_heads, near = B / 2;
  std::vector<int> row;
  for (int n = 0; row.empty() || row.back() < B - 1; ++n)
    row.push_back(n < near ? n : std::min(B - 1, near + (int)std::floor(std::log((double)n / near) / std::log((double)l.s.rel_reach / near) * (B - near))));
  l.dist_len = (int)row.size();
  std::vector<float> v((size_t)H * l.dist_len);
  for (int h = 0; h < H; ++h)
    for (int n = 0; n < l.dist_len; ++n) v[(size_t)h * l.dist_len + n] = (float)(table[(size_t)row[n] * H + h] * kLog2e);
  return upload_f32(v, &l.dist);
}

b200_status take_floats(b200_decoder* m, int layer, int which, std::vector<float>* out) {
  std::vector<uint16_t> bits;
  b200_status st = take(m, layer, which, &bits);
  out->clear();
  for (uint16_t b : bits) out->push_back(bf16_to_f(b));
  return st;
}

}  // namespace

extern "C" {

b200_status b200_decoder_create(const b200_decoder_config* c, const b200_decoder_layer* layers, b200_decoder** out) {
  *out = nullptr;
  b200_status st = b200_require_device();
  if (st != B200_OK) return st;
  const bool loop = c->loop_times > 0;
  if (c->n_layers <= 0 || c->hidden <= 0 || c->vocab <= 0 || c->max_rows <= 0 || c->max_reqs <= 0 || c->max_seqs <= 0 ||
      (c->dtype != B200_DT_BF16 && c->dtype != B200_DT_F32) ||
      (loop && (c->flags & (B200_DEC_DEPTH_AVERAGE | B200_DEC_SUM_NORM))) || ((c->flags & B200_DEC_DEPTH_AVERAGE) && (c->flags & B200_DEC_SUM_NORM)) ||
      (loop && (c->loop_start < 0 || c->loop_stop > c->n_layers || c->loop_start >= c->loop_stop))) {
    b200_set_error("decoder: invalid configuration");
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (c->hidden > 48 * 1024) { b200_set_error("decoder: width %d is larger than a row buffer", c->hidden); return B200_ERR_UNSUPPORTED; }
  auto* m = new b200_decoder();
  m->cfg = *c;
  m->layers.resize(c->n_layers);
  size_t qw = 0, yw = pad64(c->hidden), aw = 0, fw = 0, plain_w = 0, lat_w = 0, assign = 0, moe_aw = 0, ql_w = 0, lru_w = 0, mem_w = 0;
  int taps = 0;
  bool gated = false;
  for (int i = 0; i < c->n_layers; ++i) {
    const b200_decoder_layer& s = layers[i];
    bool good = s.n_heads > 0 && s.key_dim > 0 && s.value_dim > 0 && s.ffn >= 0 && s.window >= 0 && s.n_experts >= 0;
    if (s.mixer == B200_MIX_ATTENTION)
      good = good && s.n_kv_heads > 0 && s.n_heads % s.n_kv_heads == 0 && s.conv_taps >= 0 && s.rot_dim >= 0 && s.rot_dim % 2 == 0 && s.rot_dim <= s.key_dim &&
             s.q_temp_every >= 0 &&
             (!(s.flags & B200_DEC_QK_NORM_WEIGHT) || (s.flags & B200_DEC_QK_NORM)) && !((s.flags & B200_DEC_SINK) && (s.flags & B200_DEC_SINK_ONE));
    else
      good = good && s.mem_heads == 0 && !(s.flags & (B200_DEC_SINK_ONE | B200_DEC_QK_NORM_WEIGHT | B200_DEC_QK_NORM_ROW)) && s.rel_buckets == 0 && s.q_temp_every == 0;
    if (s.rel_buckets != 0) good = good && s.rel_buckets >= 2 && s.rel_reach > s.rel_buckets / 2 && !(s.flags & B200_DEC_DISTANCE_BIAS);
    if (s.mixer == B200_MIX_ATTENTION && ((s.flags & B200_DEC_QK_NORM_ROW) || s.q_temp_every > 0 || s.kv_source != 0))  // (decoder_qkv_row_kernel)
      good = good && s.conv_taps == 0 && s.rot_dim == 0 && s.mem_heads == 0 && !(s.flags & B200_DEC_QK_NORM);
    good = good && s.input_taps >= 0 && s.ff_limit >= 0.f && !((s.flags & B200_DEC_FF_GELU) && (s.flags & B200_DEC_FF_RELU2));
    if (s.input_taps > 0 || (s.flags & B200_DEC_RESULT_GATE)) good = good && !(c->flags & B200_DEC_SUM_NORM);
    if (s.flags & B200_DEC_RESULT_GATE) good = good && !(s.flags & B200_DEC_PARALLEL);
    if (s.flags & B200_DEC_ROUTER_PLAIN) good = good && (s.flags & B200_DEC_ROUTER);
    if (s.flags & B200_DEC_SHARED_GATE) good = good && (s.flags & B200_DEC_ROUTER) && s.n_experts > 0 && s.ffn > 0;
    if (s.mixer == B200_MIX_ATTENTION && s.mem_heads != 0) good = good && s.mem_heads > 0 && s.mem_key_dim > 0 && s.mem_value_dim > 0 && s.mem_gate_cap > 0.f;
    if (s.rot_dim > 0)
      good = good && s.rot_base > 1.0 && (s.yarn_factor == 0.0 || (s.yarn_factor > 0.0 && s.yarn_original > 0.0 && s.yarn_fast > 0.0 && s.yarn_slow > 0.0));
    if (s.kv_source != 0) {
      const int src = s.kv_source - 1;
      good = good && !loop && src >= 0 && src < i && layers[src].mixer == s.mixer && layers[src].kv_source == 0;
      if (s.mixer == B200_MIX_ATTENTION)
        good = good && layers[src].n_kv_heads == s.n_kv_heads && layers[src].key_dim == s.key_dim && layers[src].value_dim == s.value_dim;
      else
        good = good && s.mixer == B200_MIX_LATENT && layers[src].kv_rank == s.kv_rank && layers[src].rot_dim == s.rot_dim;
    }
    if (s.mixer == B200_MIX_ATTENTION) {}
    else if (s.mixer == B200_MIX_LRU) good = good && s.conv_taps > 0 && s.lru_decay > 0.f && s.window == 0 && !(s.flags & (B200_DEC_QKV_BIAS | B200_DEC_QK_NORM | B200_DEC_DISTANCE_BIAS | B200_DEC_SINK));
    else if (s.mixer == B200_MIX_LATENT) good = good && s.kv_rank > 0 && s.rot_dim >= 0 && s.rot_dim % 2 == 0 && s.q_rank >= 0 && !(s.flags & (B200_DEC_QKV_BIAS | B200_DEC_QK_NORM | B200_DEC_DISTANCE_BIAS));
    else if (s.mixer == B200_MIX_GLA) good = good && s.decay_rank > 0 && s.decay_tau > 0.f && s.window == 0 && !(s.flags & (B200_DEC_QKV_BIAS | B200_DEC_QK_NORM | B200_DEC_DISTANCE_BIAS | B200_DEC_SINK));
    else if (s.mixer == B200_MIX_DELTA) good = good && s.n_kv_heads > 0 && s.n_heads % s.n_kv_heads == 0 && s.conv_taps > 0 && s.window == 0 && !(s.flags & (B200_DEC_QKV_BIAS | B200_DEC_QK_NORM | B200_DEC_DISTANCE_BIAS | B200_DEC_SINK));
    else good = false;
    if (s.n_experts > 0) good = good && s.top_k > 0 && s.top_k <= s.n_experts && s.n_experts <= b200_moe_max_experts() && s.expert_ffn > 0;
    if (s.n_experts > 0 && s.flags & B200_DEC_ROUTER)
      good = good && s.top_k <= b200_moe_max_top() && s.n_groups >= 0 && s.n_groups <= b200_moe_max_groups() &&
             (s.n_groups == 0 || (s.n_experts % s.n_groups == 0 && s.keep_groups > 0 && s.keep_groups <= s.n_groups && s.top_k <= s.keep_groups * (s.n_experts / s.n_groups)));
    if (s.flags & B200_DEC_PARALLEL) good = good && !(s.flags & B200_DEC_POST_NORM);
    if (c->flags & B200_DEC_SUM_NORM) good = good && !(s.flags & (B200_DEC_POST_NORM | B200_DEC_PARALLEL));
    if (!good) {
      b200_set_error("decoder: layer %d has an invalid shape", i);
      delete m;
      return B200_ERR_INVALID_ARGUMENT;
    }
    b200_decoder::Layer& l = m->layers[i];
    l.s = s;
    l.hidden = c->hidden;
    taps = std::max(taps, s.input_taps);
    gated = gated || (s.flags & B200_DEC_RESULT_GATE);
    qw = std::max(qw, (size_t)s.n_heads * (s.mixer == B200_MIX_LATENT ? l.latent_width() : (s.key_dim + 15) / 16 * 16));
    yw = std::max({yw, (size_t)pad64(l.qkv_n()), (size_t)pad64(l.router_n() + 1), (size_t)pad64(2 * s.mem_heads), (size_t)(s.q_rank > 0 ? pad64(l.q_n()) : 0)});
    aw = std::max(aw, (size_t)l.out_k());
    fw = std::max(fw, (size_t)pad64(s.ffn));
    if (s.mixer == B200_MIX_LATENT) {
      plain_w = std::max(plain_w, (size_t)s.n_heads * l.plain_stride());
      lat_w = std::max(lat_w, (size_t)s.n_heads * pad64(s.kv_rank));
      ql_w = std::max(ql_w, (size_t)pad64(s.q_rank));
    }
    if (s.mixer == B200_MIX_LRU) {
      plain_w = std::max(plain_w, (size_t)s.n_heads * l.lru_group());
      lru_w = std::max(lru_w, (size_t)2 * l.attn_n());
    }
    if (s.rot_dim > 0 && (s.mixer == B200_MIX_LATENT || s.mixer == B200_MIX_ATTENTION)) {
      for (size_t t = 0; t < m->rotations.size() && l.rotation < 0; ++t) {
        const b200_decoder::Rotation& R = m->rotations[t];
        if (R.base == s.rot_base && R.dims == s.rot_dim && R.factor == s.yarn_factor && R.original == s.yarn_original && R.fast == s.yarn_fast && R.slow == s.yarn_slow)
          l.rotation = (int)t;
      }
      if (l.rotation < 0) {
        l.rotation = (int)m->rotations.size();
        m->rotations.push_back({s.rot_base, s.yarn_factor, s.yarn_original, s.yarn_fast, s.yarn_slow, s.rot_dim, nullptr, nullptr});
      }
    }
    if (s.mem_heads > 0) {
      m->has_gla = true;
      mem_w = std::max(mem_w, (size_t)s.mem_heads);
      if (b200_gla_takes_chunks(s.mem_key_dim, s.mem_value_dim, (int)m->elem())) m->gla.need(s.mem_heads, s.mem_key_dim, b200_memory_width(s.mem_value_dim));
    }
    if (s.mixer == B200_MIX_GLA) {
      m->has_gla = true;
      if (b200_gla_takes_chunks(s.key_dim, s.value_dim, (int)m->elem())) m->gla.need(s.n_heads, s.key_dim, s.value_dim);
    }
    if (l.delta()) {
      m->has_gla = true;
      m->gla.need_delta(s.n_heads, s.n_kv_heads, s.key_dim, s.value_dim, b200_gla_takes_chunks(s.key_dim, s.value_dim, (int)m->elem()));
    }
    if (s.n_experts > 0) {
      l.moe = (int)m->moe_layers.size();
      m->moe_layers.push_back(i);
      assign = std::max(assign, (size_t)s.top_k);
      moe_aw = std::max(moe_aw, (size_t)s.top_k * pad64(s.expert_ffn));
    }
  }
  const int lo = loop ? c->loop_start : 0, hi = loop ? c->loop_stop : 0;
  for (int i = 0; i < lo; ++i) m->runs.push_back({i, false});
  for (int p = 0; p < c->loop_times && loop; ++p) for (int i = lo; i < hi; ++i) m->runs.push_back({i, i == lo});
  for (int i = hi; i < c->n_layers; ++i) m->runs.push_back({i, false});
  m->hp = pad64(c->hidden);
  m->catp = pad64(2 * c->hidden);
  st = m->alloc_step(c->vocab, c->max_rows, c->max_reqs, c->max_seqs, true);
  const size_t R = c->max_rows, e = m->elem();
  auto alloc = [&](void** p, size_t bytes) {
    if (st != B200_OK || bytes == 0) return;
    if (cudaMalloc(p, bytes) != cudaSuccess || cudaMemset(*p, 0, bytes) != cudaSuccess) {  // zero: padding columns stay finite
      b200_set_error("decoder: cudaMalloc(%zu) failed", bytes);
      st = B200_ERR_CUDA;
    }
  };
  alloc((void**)&m->embed, (size_t)c->vocab * c->hidden * 2);
  alloc((void**)&m->x, R * c->hidden * 4);
  if (loop) {
    alloc((void**)&m->x0, R * c->hidden * 4);
    alloc(&m->cat, R * m->catp * e);
  }
  if (c->max_positions > 0) {
    alloc((void**)&m->pos_embed, (size_t)c->max_positions * c->hidden * 2);
    m->max_positions = c->max_positions;
  }
  alloc(&m->h, R * m->hp * e);
  if (taps > 0) alloc(&m->hc, R * m->hp * e);
  if (gated) alloc(&m->gate_y, R * m->hp * e);
  alloc(&m->y, std::max(R * yw, (size_t)c->max_reqs * 64) * e);
  alloc(&m->q, R * qw * e);
  alloc(&m->attn, R * aw * e);
  alloc(&m->act, R * fw * e);
  alloc(&m->last, (size_t)c->max_reqs * m->hp * e);
  alloc(&m->q_plain, R * plain_w * e);
  alloc(&m->lat_out, R * lat_w * e);
  alloc(&m->q_latent, R * ql_w * e);
  alloc((void**)&m->lru_gates, R * lru_w * 4);
  alloc((void**)&m->mem_gates, R * mem_w * sizeof(float4));
  if (c->flags & B200_DEC_DEPTH_AVERAGE) alloc((void**)&m->hist, (size_t)(c->n_layers + 1) * R * c->hidden * 4);
  for (b200_decoder::Rotation& t : m->rotations) {
    std::vector<double> f(t.dims / 2);
    for (int i = 0; i < t.dims / 2; ++i) f[i] = std::pow(t.base, -2.0 * i / t.dims);
    if (t.factor > 0) {
      auto dim_of = [&](double turns) { return t.dims * std::log(t.original / (6.283185307179586476925286766559 * turns)) / (2.0 * std::log(t.base)); };
      const double lo = std::max(std::floor(dim_of(t.fast)), 0.0), hi = std::min(std::ceil(dim_of(t.slow)), t.dims - 1.0);
      for (int i = 0; i < t.dims / 2; ++i) {
        const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
        f[i] = f[i] / t.factor * ramp + f[i] * (1.0 - ramp);
      }
    }
    alloc((void**)&t.freq, sizeof(double) * f.size());
    alloc((void**)&t.rows, sizeof(float2) * R * f.size());
    if (st == B200_OK) cudaMemcpy(t.freq, f.data(), sizeof(double) * f.size(), cudaMemcpyHostToDevice);
  }
  if (!m->moe_layers.empty()) {
    if (!m->f32()) alloc(&m->moe_x, R * assign * m->hp * e);
    alloc(&m->moe_act, R * moe_aw * e);
    alloc(&m->moe_y, R * assign * m->hp * e);
    alloc((void**)&m->moe_wts, R * assign * 4);
    alloc((void**)&m->shared_w, R * 4);
    for (int i : m->moe_layers) {
      const b200_decoder_layer& s = m->layers[i].s;
      const size_t A = R * s.top_k;
      MoeTableLayer t;
      t.n_experts = s.n_experts;
      t.top = s.top_k;
      alloc((void**)&t.indices, 4 * A + 16);
      alloc((void**)&t.offsets, 4 * (s.n_experts + 1));
      alloc((void**)&t.order, 4 * A);
      alloc((void**)&t.inv_order, 4 * A);
      alloc((void**)&t.n_items, 4);
      alloc((void**)&t.items, sizeof(int4) * (s.n_experts + A / 16 + 1));
      m->moe.push_back(t);
    }
  }
  if (m->has_gla && st == B200_OK) {
    m->gla.max_rows = c->max_rows;
    m->gla.max_reqs = c->max_reqs;
    if (!m->gla.alloc()) { b200_set_error("decoder: no memory for the chunks of %d rows", c->max_rows); st = B200_ERR_CUDA; }
  }
  if (st != B200_OK) { delete m; return st; }
  *out = m;
  return B200_OK;
}

void b200_decoder_destroy(b200_decoder* m) { delete m; }
b200_model* b200_decoder_model(b200_decoder* m) { return m; }

b200_status b200_decoder_set_tensor(b200_decoder* m, int32_t layer, int32_t which, const void* h_bf16, uint64_t n) {
  if (which < 0 || which > B200_DEC_LAST_TENSOR || (!global_tensor(which) && (layer < 0 || layer >= m->cfg.n_layers))) {
    b200_set_error("decoder: no tensor %d in layer %d", which, layer);
    return B200_ERR_INVALID_ARGUMENT;
  }
  const uint64_t want = tensor_elems(m, layer, which);
  if (want != n) {
    b200_set_error("decoder: the %s tensor of layer %d has %llu elements, the configuration asks for %llu", kTensorNames[which], layer,
                   (unsigned long long)n, (unsigned long long)want);
    return B200_ERR_INVALID_ARGUMENT;
  }
  m->staged[{global_tensor(which) ? -1 : layer, which}].bits.assign((const uint16_t*)h_bf16, (const uint16_t*)h_bf16 + n);
  return B200_OK;
}

b200_status b200_decoder_set_table(b200_decoder* m, int32_t layer, const int32_t* h_table, uint64_t n) {
  if (layer < 0 || layer >= m->cfg.n_layers || m->layers[layer].s.n_experts <= 0 || n != (uint64_t)m->cfg.vocab * m->layers[layer].s.top_k) {
    b200_set_error("decoder: an expert table of %llu numbers for layer %d", (unsigned long long)n, layer);
    return B200_ERR_INVALID_ARGUMENT;
  }
  for (uint64_t i = 0; i < n; ++i)
    if (h_table[i] < 0 || h_table[i] >= m->layers[layer].s.n_experts) {
      b200_set_error("decoder: the expert table of layer %d names expert %d of %d", layer, h_table[i], m->layers[layer].s.n_experts);
      return B200_ERR_INVALID_ARGUMENT;
    }
  m->layers[layer].h_table.assign(h_table, h_table + n);
  return B200_OK;
}

b200_status b200_decoder_finalize(b200_decoder* m) {
  const b200_decoder_config& c = m->cfg;
  b200_status st;
  for (int i = 0; i < c.n_layers; ++i) {
    b200_decoder::Layer& l = m->layers[i];
    const b200_decoder_layer& s = l.s;
    if ((st = take_weight(m, i, l.projections(), c.hidden, false, &l.wqkv)) != B200_OK) return st;
    std::vector<std::pair<int, int>> beside{{B200_DEC_W_O, l.attn_n()}};
    if (s.mem_heads > 0) beside.push_back({B200_DEC_W_MEM_O, l.mem_n()});
    if (l.parallel() && s.ffn > 0) beside.push_back({B200_DEC_W_DOWN, s.ffn});
    if (beside.size() > 1) st = take_beside(m, i, beside, c.hidden, &l.wo);
    else st = take_weight(m, i, {B200_DEC_W_O}, l.attn_n(), false, &l.wo);
    if (st != B200_OK) return st;
    if ((st = take_norm(m, i, B200_DEC_NORM1, &l.norm1)) != B200_OK) return st;
    if (s.flags & B200_DEC_POST_NORM) if ((st = take_norm(m, i, B200_DEC_POSTNORM1, &l.post1)) != B200_OK) return st;
    if (s.ffn > 0) {
      st = l.plain_ff() ? take_weight(m, i, {B200_DEC_W_UP}, c.hidden, false, &l.wgu) : take_weight(m, i, {B200_DEC_W_GATE, B200_DEC_W_UP}, c.hidden, true, &l.wgu);
      if (st != B200_OK) return st;
      if (!l.parallel()) if ((st = take_weight(m, i, {B200_DEC_W_DOWN}, s.ffn, false, &l.wdown)) != B200_OK) return st;
    }
    if (s.n_experts > 0) {
      if ((st = take_experts(m, i, l)) != B200_OK) return st;
      std::vector<int> rows{B200_DEC_W_ROUTER};
      if (l.shared_gate()) rows.push_back(B200_DEC_W_SHARED_GATE);
      st = s.flags & B200_DEC_ROUTER ? take_weight(m, i, rows, c.hidden, false, &l.wrouter) : upload_table(m, i, l);
      if (st != B200_OK) return st;
    }
    if ((s.ffn > 0 || s.n_experts > 0) && !l.parallel()) {
      if ((st = take_norm(m, i, B200_DEC_NORM2, &l.norm2)) != B200_OK) return st;
      if (s.flags & B200_DEC_POST_NORM) if ((st = take_norm(m, i, B200_DEC_POSTNORM2, &l.post2)) != B200_OK) return st;
    }
    if (c.flags & B200_DEC_DEPTH_AVERAGE) if ((st = take_vector(m, i, B200_DEC_DEPTH, &l.depth)) != B200_OK) return st;
    if (s.mixer == B200_MIX_LATENT) {
      if (s.kv_source == 0) if ((st = take_vector(m, i, B200_DEC_DKV_NORM, &l.dkv_norm)) != B200_OK) return st;
      if (s.q_rank > 0) {
        if ((st = take_vector(m, i, B200_DEC_DQ_NORM, &l.dq_norm)) != B200_OK) return st;
        if ((st = take_weight(m, i, {B200_DEC_W_Q}, s.q_rank, false, &l.wuq)) != B200_OK) return st;
      }
      if ((st = take_stack(m, i, B200_DEC_W_UK, s.n_heads, s.kv_rank, s.key_dim, true, &l.wuk)) != B200_OK) return st;
      if ((st = take_stack(m, i, B200_DEC_W_UV, s.n_heads, s.value_dim, s.kv_rank, false, &l.wuv)) != B200_OK) return st;
    }
    if (s.mixer == B200_MIX_GLA) {
      if ((st = take_vector(m, i, B200_DEC_W_A2, &l.a2)) != B200_OK) return st;
      if ((st = take_vector(m, i, B200_DEC_B_A2, &l.a2_bias)) != B200_OK) return st;
      if ((st = take_vector(m, i, B200_DEC_HEAD_NORM, &l.head_norm)) != B200_OK) return st;
    }
    if (s.flags & B200_DEC_QKV_BIAS) {
      if ((st = take_vectors(m, i, {B200_DEC_B_Q, B200_DEC_B_K, B200_DEC_B_V}, &l.bias)) != B200_OK) return st;
    }
    if (s.flags & B200_DEC_QK_NORM_WEIGHT) {
      if ((st = take_vector(m, i, B200_DEC_Q_NORM, &l.q_norm)) != B200_OK) return st;
      if ((st = take_vector(m, i, B200_DEC_K_NORM, &l.k_norm)) != B200_OK) return st;
    }
    if (s.flags & B200_DEC_QK_NORM_ROW) {
      if ((st = take_vector(m, i, B200_DEC_Q_NORM, &l.q_norm)) != B200_OK) return st;
      if (s.kv_source == 0) if ((st = take_vector(m, i, B200_DEC_K_NORM, &l.k_norm)) != B200_OK) return st;
    }
    std::vector<float> v;
    if (s.rel_buckets > 0)
      if ((st = take_floats(m, i, B200_DEC_W_REL, &v)) != B200_OK || (st = make_distances(l, v)) != B200_OK) return st;
    const int subs = l.second() ? 2 : 1;
    for (int w = 0; w < subs && s.input_taps > 0; ++w)
      if ((st = take_conv(m, i, {w ? B200_DEC_IN_CONV2 : B200_DEC_IN_CONV1}, s.input_taps, &l.in_conv[w])) != B200_OK) return st;
    for (int w = 0; w < subs && s.flags & B200_DEC_RESULT_GATE; ++w) {
      if ((st = take_weight(m, i, {w ? B200_DEC_W_RESULT_GATE2 : B200_DEC_W_RESULT_GATE1}, c.hidden, false, &l.wgate[w])) != B200_OK) return st;
      if ((st = take_vector(m, i, w ? B200_DEC_B_RESULT_GATE2 : B200_DEC_B_RESULT_GATE1, &l.out_gate_bias[w])) != B200_OK) return st;
    }
    if (l.delta()) {
      if ((st = take_vector(m, i, B200_DEC_DT_BIAS, &l.dt_bias)) != B200_OK || (st = take_vector(m, i, B200_DEC_HEAD_NORM, &l.head_norm)) != B200_OK ||
          (st = take_floats(m, i, B200_DEC_A_LOG, &v)) != B200_OK)
        return st;
      for (float& x : v) x = (float)std::exp((double)x);
      if ((st = upload_f32(v, &l.rate)) != B200_OK) return st;
    }
    if ((s.mixer == B200_MIX_ATTENTION || l.delta()) && s.conv_taps > 0)
      if ((st = take_conv(m, i, {B200_DEC_CONV_Q, B200_DEC_CONV_K, B200_DEC_CONV_V}, s.conv_taps, &l.conv)) != B200_OK) return st;
    if (s.mem_heads > 0) {
      if ((st = take_weight(m, i, {B200_DEC_W_MEM_I, B200_DEC_W_MEM_F}, c.hidden, false, &l.wgates)) != B200_OK) return st;
      if ((st = take_vectors(m, i, {B200_DEC_B_MEM_I, B200_DEC_B_MEM_F}, &l.gate_bias)) != B200_OK) return st;
      if ((st = take_vector(m, i, B200_DEC_MEM_NORM, &l.mem_norm)) != B200_OK) return st;
    }
    if (s.mixer == B200_MIX_LRU) {
      if ((st = take_vectors(m, i, {B200_DEC_B_LRU_Y, B200_DEC_B_LRU_X, B200_DEC_B_LRU_R, B200_DEC_B_LRU_I}, &l.lru_bias)) != B200_OK) return st;
      if ((st = take_conv(m, i, {B200_DEC_LRU_CONV}, s.conv_taps, &l.conv)) != B200_OK) return st;
      if ((st = take_vector(m, i, B200_DEC_B_LRU_CONV, &l.conv_bias)) != B200_OK) return st;
      if ((st = take_lru(m, i, l)) != B200_OK) return st;
    }
    if (s.flags & B200_DEC_SINK_ONE) if ((st = upload_f32(std::vector<float>(s.n_heads, 0.f), &l.sinks)) != B200_OK) return st;
    if (s.flags & B200_DEC_SINK) if ((st = take_vector(m, i, B200_DEC_W_SINK, &l.sinks, kLog2e)) != B200_OK) return st;
    if ((st = make_slopes(l)) != B200_OK) return st;
  }
  if (c.loop_times > 0) if ((st = take_weight(m, -1, {B200_DEC_W_LOOP_IN}, 2 * c.hidden, false, &m->loop_in)) != B200_OK) return st;
  if ((st = take_weight(m, -1, {B200_DEC_W_HEAD}, c.hidden, false, &m->head)) != B200_OK) return st;
  // (the logits' scale rides on the final norm's weight)
  if ((st = take_norm(m, -1, B200_DEC_FINAL_NORM, &m->final_norm, c.logit_scale)) != B200_OK) return st;
  if ((st = upload_moe(m)) != B200_OK) return st;
  std::vector<uint16_t> table;
  if (c.max_positions > 0) {
    if ((st = take(m, -1, B200_DEC_W_POS, &table)) != B200_OK) return st;
    B200_CUDA_TRY(cudaMemcpy(m->pos_embed, table.data(), table.size() * 2, cudaMemcpyHostToDevice));
  }
  if ((st = take(m, -1, B200_DEC_W_EMBED, &table)) != B200_OK) return st;
  B200_CUDA_TRY(cudaMemcpy(m->embed, table.data(), table.size() * 2, cudaMemcpyHostToDevice));
  m->ready = true;
  return B200_OK;
}

b200_status b200_decoder_random_init(b200_decoder* m, uint32_t seed) {
  const b200_decoder_config& c = m->cfg;
  b200_status st;
  const std::vector<float> ones(c.hidden, 1.f);
  auto stack = [&](int count, int n, int k, uint32_t salt, b200_qweight** out) -> b200_status {
    if (n % 64 || k % 64) { b200_set_error("random_init: a %d x %d projection (multiples of 64 only)", n, k); return B200_ERR_INVALID_ARGUMENT; }
    return b200_qweight_random(B200_Q_BF16, count, n, k, seed + salt, out);
  };
  auto weight = [&](int n, int k, uint32_t salt, b200_qweight** out) -> b200_status { return stack(1, n, k, salt, out); };
  for (int i = 0; i < c.n_layers; ++i) {
    b200_decoder::Layer& l = m->layers[i];
    const b200_decoder_layer& s = l.s;
    if ((st = weight(pad64(l.qkv_n()), c.hidden, 16 * i + 1, &l.wqkv)) != B200_OK) return st;
    if ((st = weight(c.hidden, l.out_k(), 16 * i + 2, &l.wo)) != B200_OK) return st;
    if ((st = upload_f32(ones, &l.norm1)) != B200_OK) return st;
    if (s.flags & B200_DEC_POST_NORM) if ((st = upload_f32(ones, &l.post1)) != B200_OK) return st;
    if (s.ffn > 0) {
      if ((st = weight((l.plain_ff() ? 1 : 2) * s.ffn, c.hidden, 16 * i + 3, &l.wgu)) != B200_OK) return st;
      if (!l.parallel()) if ((st = weight(c.hidden, s.ffn, 16 * i + 4, &l.wdown)) != B200_OK) return st;
    }
    if ((s.ffn > 0 || s.n_experts > 0) && !l.parallel()) {
      if ((st = upload_f32(ones, &l.norm2)) != B200_OK) return st;
      if (s.flags & B200_DEC_POST_NORM) if ((st = upload_f32(ones, &l.post2)) != B200_OK) return st;
    }
    if (s.n_experts > 0) {
      if ((st = stack(s.n_experts, (l.plain_ff() ? 1 : 2) * s.expert_ffn, c.hidden, 16 * i + 5, &l.we_gu)) != B200_OK) return st;
      if ((st = stack(s.n_experts, c.hidden, s.expert_ffn, 16 * i + 6, &l.we_down)) != B200_OK) return st;
      if (s.flags & B200_DEC_ROUTER) {
        if ((st = weight(pad64(s.n_experts + (l.shared_gate() ? 1 : 0)), c.hidden, 16 * i + 9, &l.wrouter)) != B200_OK) return st;
      } else {
      l.h_table.resize((size_t)c.vocab * s.top_k);
      uint32_t x = seed * 747796405u + i;
      for (int v = 0; v < c.vocab; ++v) {  // experts an odd step apart from a random one: all different
        x = x * 1664525u + 1013904223u;
        for (int j = 0; j < s.top_k; ++j) l.h_table[(size_t)v * s.top_k + j] = (int)(((x >> 8) + (uint32_t)j) % (uint32_t)s.n_experts);
      }
      if ((st = upload_table(m, i, l)) != B200_OK) return st;
      }
    }
    if (c.flags & B200_DEC_DEPTH_AVERAGE) {
      std::vector<float> d(i + 2, 0.1f);
      d[i + 1] = 0.8f;
      if ((st = upload_f32(d, &l.depth)) != B200_OK) return st;
    }
    if (s.mixer == B200_MIX_LATENT) {
      if (s.kv_source == 0) if ((st = upload_f32(std::vector<float>(s.kv_rank, 1.f), &l.dkv_norm)) != B200_OK) return st;
      if (s.q_rank > 0) {
        if ((st = upload_f32(std::vector<float>(s.q_rank, 1.f), &l.dq_norm)) != B200_OK) return st;
        if ((st = weight(pad64(l.q_n()), s.q_rank, 16 * i + 10, &l.wuq)) != B200_OK) return st;
      }
      if ((st = stack(s.n_heads, s.kv_rank, l.plain_stride(), 16 * i + 7, &l.wuk)) != B200_OK) return st;
      if ((st = stack(s.n_heads, s.value_dim, pad64(s.kv_rank), 16 * i + 8, &l.wuv)) != B200_OK) return st;
    }
    if (s.mixer == B200_MIX_GLA) {
      if ((st = upload_f32(std::vector<float>((size_t)s.n_heads * s.key_dim * s.decay_rank, 0.02f), &l.a2)) != B200_OK) return st;
      if ((st = upload_f32(std::vector<float>((size_t)s.n_heads * s.key_dim, 2.f), &l.a2_bias)) != B200_OK) return st;
      if ((st = upload_f32(std::vector<float>(s.value_dim, 1.f), &l.head_norm)) != B200_OK) return st;
    }
    if (s.flags & B200_DEC_QKV_BIAS) if ((st = upload_f32(std::vector<float>(l.qkv_n(), 0.01f), &l.bias)) != B200_OK) return st;
    if (s.flags & B200_DEC_SINK) if ((st = upload_f32(std::vector<float>(s.n_heads, 0.5f), &l.sinks)) != B200_OK) return st;
    auto fill = [&](size_t n, float v, float** out) { return upload_f32(std::vector<float>(n, v), out); };
    if (s.flags & B200_DEC_SINK_ONE) if ((st = fill(s.n_heads, 0.f, &l.sinks)) != B200_OK) return st;
    if (s.flags & B200_DEC_QK_NORM_WEIGHT)
      if ((st = fill(s.key_dim, 1.f, &l.q_norm)) != B200_OK || (st = fill(s.key_dim, 1.f, &l.k_norm)) != B200_OK) return st;
    if (s.mixer == B200_MIX_ATTENTION && s.conv_taps > 0) if ((st = upload_bf16(std::vector<uint16_t>((size_t)l.attention_n() * s.conv_taps, 0x3F00), &l.conv)) != B200_OK) return st;
    if (s.flags & B200_DEC_QK_NORM_ROW)
      if ((st = fill((size_t)s.n_heads * s.key_dim, 1.f, &l.q_norm)) != B200_OK || (st = fill((size_t)s.n_kv_heads * s.key_dim, 1.f, &l.k_norm)) != B200_OK) return st;
    if (s.rel_buckets > 0) if ((st = make_distances(l, std::vector<float>((size_t)s.rel_buckets * s.n_heads, 0.25f))) != B200_OK) return st;
    for (int w = 0; w < (l.second() ? 2 : 1); ++w) {
      if (s.input_taps > 0) if ((st = upload_bf16(std::vector<uint16_t>((size_t)c.hidden * s.input_taps, 0x3E80), &l.in_conv[w])) != B200_OK) return st;
      if (s.flags & B200_DEC_RESULT_GATE)
        if ((st = weight(c.hidden, c.hidden, 16 * i + 13 + w, &l.wgate[w])) != B200_OK || (st = fill(c.hidden, 0.1f, &l.out_gate_bias[w])) != B200_OK) return st;
    }
    if (l.delta()) {
      const size_t channels = b200_delta_channels(s.n_heads, s.n_kv_heads, s.key_dim, s.value_dim);
      if ((st = upload_bf16(std::vector<uint16_t>(channels * s.conv_taps, 0x3F00), &l.conv)) != B200_OK || (st = fill(s.n_heads, 0.5f, &l.rate)) != B200_OK ||
          (st = fill(s.n_heads, -2.f, &l.dt_bias)) != B200_OK || (st = fill(s.value_dim, 1.f, &l.head_norm)) != B200_OK)
        return st;
    }
    if (s.mem_heads > 0) {
      if ((st = weight(pad64(2 * s.mem_heads), c.hidden, 16 * i + 11, &l.wgates)) != B200_OK) return st;
      if ((st = fill(2 * s.mem_heads, 1.f, &l.gate_bias)) != B200_OK || (st = fill(l.mem_n(), 1.f, &l.mem_norm)) != B200_OK) return st;
    }
    if (s.mixer == B200_MIX_LRU) {
      if ((st = stack(s.n_heads, 2 * s.value_dim, l.lru_group(), 16 * i + 12, &l.wgates)) != B200_OK) return st;
      if ((st = fill(4 * l.attn_n(), 0.1f, &l.lru_bias)) != B200_OK || (st = upload_bf16(std::vector<uint16_t>((size_t)l.attn_n() * s.conv_taps, 0x3F00), &l.conv)) != B200_OK ||
          (st = fill(l.attn_n(), 0.f, &l.conv_bias)) != B200_OK || (st = fill(l.attn_n(), 0.5f, &l.lru_rate)) != B200_OK)
        return st;
    }
    if ((st = make_slopes(l)) != B200_OK) return st;
  }
  if ((st = upload_moe(m)) != B200_OK) return st;
  if (c.loop_times > 0) if ((st = weight(c.hidden, 2 * c.hidden, 11, &m->loop_in)) != B200_OK) return st;
  if ((st = weight(c.vocab, c.hidden, 7, &m->head)) != B200_OK) return st;
  if ((st = upload_f32(ones, &m->final_norm)) != B200_OK) return st;
  std::vector<uint16_t> emb((size_t)c.vocab * c.hidden);
  uint32_t s = seed * 2654435761u + 12345u;
  for (auto& e : emb) { s = s * 1664525u + 1013904223u; e = (uint16_t)(((s >> 16) & 0x807F) | 0x3C80); }
  B200_CUDA_TRY(cudaMemcpy(m->embed, emb.data(), emb.size() * 2, cudaMemcpyHostToDevice));
  if (c.max_positions > 0) B200_CUDA_TRY(cudaMemset(m->pos_embed, 0, (size_t)c.max_positions * c.hidden * 2));
  m->ready = true;
  return B200_OK;
}

int32_t b200_decoder_cache_layers(const b200_decoder* m, b200_kv_layer* out, int32_t cap) {
  for (size_t r = 0; r < m->runs.size() && (int)r < cap; ++r) {
    out[r] = m->layers[m->runs[r].layer].cache();
  }
  return (int32_t)m->runs.size();
}

b200_status b200_decoder_record_layers(b200_decoder* m, int32_t on) {
  if (on && !m->rec) B200_CUDA_TRY(cudaMalloc((void**)&m->rec, sizeof(float) * m->runs.size() * (size_t)m->max_rows * m->cfg.hidden));
  m->recording = on != 0;
  m->drop_graphs();
  return B200_OK;
}

b200_status b200_decoder_recorded_layers(b200_decoder* m, int32_t rows, float* h_out) {
  if (!m->rec || rows < 0 || rows > m->max_rows) { b200_set_error("recorded_layers: nothing recorded, or %d rows", rows); return B200_ERR_INVALID_ARGUMENT; }
  B200_CUDA_TRY(cudaDeviceSynchronize());
  for (size_t r = 0; r < m->runs.size(); ++r)
    B200_CUDA_TRY(cudaMemcpy(h_out + r * (size_t)rows * m->cfg.hidden, m->rec + r * (size_t)m->max_rows * m->cfg.hidden,
                             sizeof(float) * (size_t)rows * m->cfg.hidden, cudaMemcpyDeviceToHost));
  return B200_OK;
}

void b200_decoder_set_attn_mma(b200_decoder* m, int32_t on) {
  m->attn_mma = on != 0;
  m->drop_graphs();
}

b200_status b200_decoder_qkv(b200_kv* kv, int32_t layer, const void* d_qkv, int32_t stride, const float* d_bias, int32_t n_q_heads,
                             int32_t qk_norm, float eps, void* d_q, const int32_t* d_positions, const int32_t* d_row_seq,
                             int32_t total_rows, void* stream) {
  if (!kv->layered || layer < 0 || layer >= kv->cfg.n_layers || n_q_heads <= 0 || kv->lay[layer].heads <= 0 || n_q_heads % kv->lay[layer].heads != 0) {
    b200_set_error("decoder_qkv: layer %d with %d query heads", layer, n_q_heads);
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (total_rows <= 0) return B200_OK;
  QkvArgs a;
  a.d = kv->dev; a.L = kv->lay[layer]; a.bias = d_bias; a.hq = n_q_heads; a.qk_norm = qk_norm; a.eps = eps; a.q = d_q;
  a.src.y = d_qkv;
  a.src.y_stride = stride;
  a.q_stride = n_q_heads * a.L.kd;
  a.pos = d_positions; a.row_seq = d_row_seq;
  return launch_qkv(a, total_rows, (cudaStream_t)stream);
}

b200_status b200_decoder_attention(b200_kv* kv, int32_t layer, const void* d_q, int32_t n_q_heads, int32_t window, float scale,
                                   const float* d_slopes_log2, const float* d_sinks_log2, const float* d_dist_log2, int32_t dist_len,
                                   const int32_t* d_row_seq, const int32_t* d_row_ctx, int32_t total_rows, int32_t mma, void* d_out,
                                   int32_t out_stride, void* stream) {
  if (!kv->layered || layer < 0 || layer >= kv->cfg.n_layers || n_q_heads <= 0 || n_q_heads > kv->cfg.n_q_heads || kv->lay[layer].heads <= 0 ||
      n_q_heads % kv->lay[layer].heads != 0 || window < 0 || (d_dist_log2 && (dist_len <= 0 || kv->lay[layer].values_in_keys))) {
    b200_set_error("decoder_attention: layer %d with %d query heads, window %d", layer, n_q_heads, window);
    return B200_ERR_INVALID_ARGUMENT;
  }
  b200_status st = B200_OK;
  if (mma && b200_window_attn_takes_mma(kv, layer))
    st = b200_window_attn_plan(kv, layer, window, n_q_heads / kv->lay[layer].heads, d_row_seq, d_row_ctx, total_rows, stream);
  if (st != B200_OK) return st;
  WindowAttnCall c;
  c.layer = layer; c.n_q_heads = n_q_heads; c.window = window; c.q = d_q; c.q_stride = n_q_heads * kv->lay[layer].kd; c.scale = scale;
  c.slopes_log2 = d_slopes_log2; c.sinks_log2 = d_sinks_log2; c.dist_log2 = d_dist_log2; c.dist_len = dist_len; c.out = d_out; c.out_stride = out_stride;
  return b200_window_attn_run(kv, c, d_row_seq, d_row_ctx, total_rows, mma != 0, stream);
}

b200_status b200_decoder_gla(b200_kv* kv, int32_t layer, const b200_gla_shape* z, const void* d_rows, int32_t stride, const float* d_a2,
                             const float* d_a2_bias, const float* d_norm, const int32_t* d_cu, const int32_t* d_row_seq,
                             const int32_t* d_positions, int32_t n_req, int32_t total_rows, int32_t chunked, void* d_out, int32_t out_stride,
                             void* stream) {
  if (n_req <= 0 || total_rows <= 0) return B200_OK;
  GlaScratch g;
  g.max_rows = total_rows;
  g.max_reqs = n_req;
  if (b200_gla_takes_chunks(z->key_dim, z->value_dim, kv->dev.elem_bytes)) g.need(z->heads, z->key_dim, z->value_dim);
  if (!g.alloc()) { g.free(); b200_set_error("decoder_gla: no memory for %d rows", total_rows); return B200_ERR_CUDA; }
  GlaCall c;
  c.layer = layer; c.heads = z->heads; c.dk = z->key_dim; c.dv = z->value_dim; c.rank = z->decay_rank;
  c.src.y = d_rows; c.src.y_stride = stride;
  c.a2 = d_a2; c.a2_bias = d_a2_bias; c.norm = d_norm; c.q_scale = z->q_scale; c.inv_tau = z->inv_tau; c.eps = z->eps;
  c.out = d_out; c.out_stride = out_stride;
  b200_status st = b200_gla_plan(g, d_cu, n_req, total_rows, stream);
  if (st == B200_OK) st = b200_gla_run(kv, g, c, d_cu, d_row_seq, d_positions, n_req, total_rows, chunked != 0, stream);
  const cudaError_t e = cudaStreamSynchronize((cudaStream_t)stream);
  g.free();
  if (st == B200_OK && e != cudaSuccess) { b200_set_error("decoder_gla: %s", cudaGetErrorString(e)); return B200_ERR_CUDA; }
  return st;
}

b200_status b200_decoder_delta(b200_kv* kv, int32_t layer, const b200_delta_shape* z, const void* d_rows, int32_t stride, const void* d_conv,
                               const float* d_rate, const float* d_dt_bias, const float* d_norm, const int32_t* d_cu, const int32_t* d_row_to_req,
                               const int32_t* d_row_seq, const int32_t* d_positions, int32_t n_req, int32_t total_rows, int32_t chunked,
                               void* d_out, int32_t out_stride, void* stream) {
  if (n_req <= 0 || total_rows <= 0) return B200_OK;
  GlaScratch g;
  g.max_rows = total_rows;
  g.max_reqs = n_req;
  g.need_delta(z->heads, z->kv_heads, z->key_dim, z->value_dim, b200_gla_takes_chunks(z->key_dim, z->value_dim, kv->dev.elem_bytes));
  if (!g.alloc()) { g.free(); b200_set_error("decoder_delta: no memory for %d rows", total_rows); return B200_ERR_CUDA; }
  DeltaCall c;
  c.layer = layer; c.heads = z->heads; c.kv_heads = z->kv_heads; c.dk = z->key_dim; c.dv = z->value_dim;
  c.src.y = d_rows; c.src.y_stride = stride;
  c.conv.taps = z->taps; c.conv.w = (const __nv_bfloat16*)d_conv;
  c.rate = d_rate; c.dt_bias = d_dt_bias; c.norm = d_norm; c.eps = z->eps; c.out = d_out; c.out_stride = out_stride;
  b200_status st = b200_gla_plan(g, d_cu, n_req, total_rows, stream);
  if (st == B200_OK) st = b200_delta_prep(kv, g, c, d_cu, d_row_to_req, d_row_seq, d_positions, total_rows, stream);
  if (st == B200_OK) st = b200_delta_run(kv, g, c, d_cu, d_row_seq, d_positions, n_req, total_rows, chunked != 0, stream);
  const cudaError_t e = cudaStreamSynchronize((cudaStream_t)stream);
  g.free();
  if (st == B200_OK && e != cudaSuccess) { b200_set_error("decoder_delta: %s", cudaGetErrorString(e)); return B200_ERR_CUDA; }
  return st;
}

}  // extern "C"
