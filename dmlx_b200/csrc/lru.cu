// Gated linear recurrent unit (Griffin's recurrent block): a diagonal recurrence with an input gate and a decay gate per channel.  The
// state lives in the pool's slot of the sequence, f32, and a sequence at position 0 starts from zero, so slots need no clearing.
//
// lru_prep_kernel stands behind the projection of both branches: bias and GELU of the one, bias and causal convolution of the other.
// lru_scan_kernel walks the tokens of a request.  Portions of a prompt are cut into one segment per warp of a block: every warp first
// walks its segment from zero, the segments' decays and sums are put together, and the second walk starts from the right state.
#include <cuda_bf16.h>

#include <algorithm>

#include "common.h"
#include "lru.cuh"

namespace {

struct LruArgs {
  LruCall c;
  float* state;  // the layer's, of slot 0
  int rec_elems, block;  // block: width of a block
  const int *cu, *row_to_req, *row_seq, *pos, *pool_state;
  int max_seqs;
};

__device__ __forceinline__ float gelu_tanh(float z) {
  return 0.5f * z * (1.0f + tanhf(0.79788456080286536f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// One thread per (R rows, VEC channels).
template <typename T, int VEC, int R>
__global__ void __launch_bounds__(256) lru_prep_kernel(LruArgs a, int rows) {
  const LruCall& c = a.c;
  const int begin = blockIdx.x * R, end = min(begin + R, rows), ch = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (ch >= c.width) return;
  const Vec<VEC> yb = load_vec<VEC>(c.y_bias + ch), xb = load_vec<VEC>(c.x_bias + ch);
#pragma unroll
  for (int r = 0; r < R; ++r) {
    if (begin + r < end) {
      Vec<VEC> y = mat_value<T, VEC>(c.src, begin + r, ch);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y.v[e] = gelu_tanh(y.v[e] + yb.v[e]);
      store_vec<VEC>((T*)c.out + (size_t)(begin + r) * c.out_stride + ch, y);
    }
  }
  if (a.pool_state[ST_ERR] != 0) return;
  auto value = [&](int row, int col) {
    Vec<VEC> v = mat_value<T, VEC>(c.src, row, c.width + col);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] += xb.v[e];
    return v;
  };
  const int b = ch / a.block, o = ch - b * a.block;
  auto put = [&](int row, const Vec<VEC>& v) {
    T* u = (T*)c.u + ((size_t)row * c.blocks + b) * c.u_group;
    store_vec<VEC>(u + o, v);
    if (o + VEC == a.block)
      for (int z = a.block; z < c.u_group; ++z) st(u + z, 0.f);
  };
  if constexpr (R > 1) {
    if (c.conv.taps == 4 && begin + R <= rows && a.row_to_req[begin] == a.row_to_req[begin + R - 1] && begin - a.cu[a.row_to_req[begin]] >= 3) {
      Vec<VEC> v[R];
      conv_values_inside<4, R, VEC>(c.conv, value, begin, ch, v);
#pragma unroll
      for (int r = 0; r < R; ++r) put(begin + r, v[r]);
      return;
    }
  }
  for (int first = begin; first < end; ++first) {
    const int req = a.row_to_req[first], r0 = a.cu[req], count = a.cu[req + 1] - r0, slot = a.row_seq[first];
    if (slot < 0 || slot >= a.max_seqs) continue;
    const int n = conv_rows(c.conv, first - r0, count);
    for (int row = first; row < first + n; ++row) put(row, conv_value<VEC>(c.conv, value, row, row - r0, a.pos[row], slot, ch));
    if (first == r0) conv_update<VEC>(c.conv, value, r0, count, slot, ch);
  }
}

// SEG = 1: a thread walks all tokens of a request for one channel; otherwise a warp's lanes are 32 channels, and the block's SEG
// warps take a segment of the tokens each.
template <typename T, int SEG>
__global__ void __launch_bounds__(SEG == 1 ? 128 : 32 * SEG) lru_scan_kernel(LruArgs a) {
  __shared__ float s_log[SEG][33], s_sum[SEG][33];
  const LruCall& c = a.c;
  const int req = blockIdx.y, lane = threadIdx.x & 31, seg = SEG == 1 ? 0 : threadIdx.x >> 5;
  const int ch = SEG == 1 ? blockIdx.x * blockDim.x + threadIdx.x : blockIdx.x * 32 + lane;
  const int r0 = a.cu[req], count = a.cu[req + 1] - r0;
  if (count <= 0 || a.pool_state[ST_ERR] != 0) return;
  const int slot = a.row_seq[r0];
  if (slot < 0 || slot >= a.max_seqs) return;
  const bool on = ch < c.width;
  const int per = (count + SEG - 1) / SEG, t0 = min(seg * per, count), t1 = min(t0 + per, count);
  const int cc = on ? ch : 0, b = cc / a.block, o = cc - b * a.block;
  const float rate = c.rate[cc], rb = c.r_bias[cc], ib = c.i_bias[cc];
  float* state = a.state + (size_t)slot * a.rec_elems + cc;
  const float s0 = a.pos[r0] == 0 ? 0.f : *state;
  constexpr int U = 4;
  // tokens t0 .. t1 - 1 from state s; `log_sum` gathers their decays
  auto walk = [&](float s, float& log_sum, bool write) {
    for (int t = t0; t < t1; t += U) {
      float u[U], gr[U], gi[U], y[U];
#pragma unroll
      for (int k = 0; k < U; ++k) {
        const int row = r0 + min(t + k, t1 - 1);
        const float* g = c.gates + (size_t)row * 2 * c.width + b * 2 * a.block + o;
        u[k] = ld((const T*)c.u + ((size_t)row * c.blocks + b) * c.u_group + o);
        gr[k] = g[0];
        gi[k] = g[a.block];
        y[k] = write ? ld((const T*)c.out + (size_t)row * c.out_stride + cc) : 0.f;
      }
#pragma unroll
      for (int k = 0; k < U; ++k) {
        if (t + k < t1) {
          const float la = -rate * sigmoid(gr[k] + rb);
          s = expf(la) * s + sqrtf(-expm1f(2.0f * la)) * sigmoid(gi[k] + ib) * u[k];
          log_sum += la;
          if (write && on) st((T*)c.out + (size_t)(r0 + t + k) * c.out_stride + cc, s * y[k]);
        }
      }
    }
    return s;
  };
  float s = s0, unused = 0.f;
  if constexpr (SEG > 1) {
    float log_sum = 0.f;
    const float sum = walk(0.f, log_sum, false);
    s_log[seg][lane] = log_sum;
    s_sum[seg][lane] = sum;
    __syncthreads();
    for (int w = 0; w < seg; ++w) s = expf(s_log[w][lane]) * s + s_sum[w][lane];
  }
  s = walk(s, unused, true);
  if (on && t0 < t1 && t1 == count) *state = s;  // (every warp has read it: the barrier above)
}

b200_status args_of(b200_kv* kv, const LruCall& c, LruArgs* a) {
  if (c.layer < 0 || c.layer >= kv->cfg.n_layers || c.blocks <= 0 || c.width % c.blocks != 0 || c.u_group < c.width / c.blocks ||
      kv->lay[c.layer].rec_elems < b200_lru_elems(c.width, c.conv.taps)) {
    b200_set_error("lru: layer %d of the pool has no state of %d channels", c.layer, c.width);
    return B200_ERR_INVALID_ARGUMENT;
  }
  a->c = c;
  a->state = kv->dev.rec_pool + kv->lay[c.layer].rec_off;
  a->rec_elems = kv->lay[c.layer].rec_elems;
  a->block = c.width / c.blocks;
  a->max_seqs = kv->dev.max_seqs;
  a->pool_state = kv->dev.state;
  a->c.conv.channels = c.width;
  a->c.conv.state = a->state + b200_lru_conv_off(c.width);
  a->c.conv.slot_elems = a->rec_elems;
  return B200_OK;
}

}  // namespace

b200_status b200_lru_prep(b200_kv* kv, LruCall c, const int32_t* d_cu, const int32_t* d_row_to_req, const int32_t* d_row_seq, const int32_t* d_pos,
                          int total_rows, void* stream) {
  if (total_rows <= 0) return B200_OK;
  LruArgs a{};
  b200_status st = args_of(kv, c, &a);
  if (st != B200_OK) return st;
  a.cu = d_cu; a.row_to_req = d_row_to_req; a.row_seq = d_row_seq; a.pos = d_pos;
  const bool v4 = a.block % 4 == 0 && c.u_group % 4 == 0 && c.out_stride % 4 == 0 && a.rec_elems % 4 == 0 && (c.src.ws || c.src.y_stride % 4 == 0);
  const int groups = v4 ? c.width / 4 : c.width, threads = std::min(256, (groups + 31) / 32 * 32);
  const bool many = total_rows >= 1024, f32 = kv->dev.elem_bytes == 4;
  auto* kernel = f32 ? (v4 ? lru_prep_kernel<float, 4, 1> : lru_prep_kernel<float, 1, 1>) : (v4 ? lru_prep_kernel<__nv_bfloat16, 4, 1> : lru_prep_kernel<__nv_bfloat16, 1, 1>);
  if (many) kernel = f32 ? (v4 ? lru_prep_kernel<float, 4, 4> : lru_prep_kernel<float, 1, 4>) : (v4 ? lru_prep_kernel<__nv_bfloat16, 4, 4> : lru_prep_kernel<__nv_bfloat16, 1, 4>);
  kernel<<<dim3(many ? (total_rows + 3) / 4 : total_rows, (groups + threads - 1) / threads), threads, 0, (cudaStream_t)stream>>>(a, total_rows);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

b200_status b200_lru_scan(b200_kv* kv, const LruCall& c, const int32_t* d_cu, const int32_t* d_row_seq, const int32_t* d_pos, int n_req, int total_rows,
                          void* stream) {
  if (n_req <= 0 || total_rows <= 0) return B200_OK;
  LruArgs a{};
  b200_status st = args_of(kv, c, &a);
  if (st != B200_OK) return st;
  a.cu = d_cu; a.row_seq = d_row_seq; a.pos = d_pos;
  const bool f32 = kv->dev.elem_bytes == 4;
  cudaStream_t s = (cudaStream_t)stream;
  if (total_rows <= 8 * n_req) {
    auto* kernel = f32 ? lru_scan_kernel<float, 1> : lru_scan_kernel<__nv_bfloat16, 1>;
    kernel<<<dim3((c.width + 127) / 128, n_req), 128, 0, s>>>(a);
  } else {
    auto* kernel = f32 ? lru_scan_kernel<float, 16> : lru_scan_kernel<__nv_bfloat16, 16>;
    kernel<<<dim3((c.width + 31) / 32, n_req), 512, 0, s>>>(a);
  }
  B200_LAUNCH_CHECK();
  return B200_OK;
}
