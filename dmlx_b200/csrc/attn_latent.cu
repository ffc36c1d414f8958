// Latent attention: all heads attend to one row per token, [latent c | rotated key part], and their values are W_uv c.  W_uk is
// taken to the query side (q_head <- W_uk^T q_head) and W_uv behind the weighted sum, so the pages are read once for all heads
// and hold kv_rank + rot_dim numbers per token.
#include <cuda_bf16.h>

#include <algorithm>

#include "attn_latent.cuh"
#include "common.h"

namespace {

// Angles in f64, brought into one turn before they become f32: positions far out keep their accuracy.
__global__ void __launch_bounds__(256) rotation_table_kernel(const double* __restrict__ freq, int half, const int* __restrict__ pos, int rows,
                                                             float2* __restrict__ out) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= (long long)rows * half) return;
  const int row = (int)(i / half), p = (int)(i - (long long)row * half);
  constexpr double kTurn = 6.283185307179586476925286766559;
  const double a = (double)pos[row] * freq[p];
  float s, c;
  sincosf((float)(a - rint(a / kTurn) * kTurn), &s, &c);
  out[i] = make_float2(c, s);
}

struct PrepArgs {
  KvDev d;
  KvLayerDev L;
  LatentPrep p;
  const int *pos, *row_seq;
};

// One warp per (row, query head), and one for the row's latent.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_prep_kernel(PrepArgs a) {
  const LatentPrep& p = a.p;
  const int row = blockIdx.x, lane = threadIdx.x & 31, u = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (u > p.heads) return;
  const int per_head = p.dim + p.rot;
  const float2* rt = p.rotation + (size_t)row * (p.rot / 2);
  auto rotate = [&](T* dst, int col) {
    for (int i = lane; i < p.rot / 2; i += 32) {
      const float x = mat_value<T, 1>(p.src, row, col + 2 * i).v[0], y = mat_value<T, 1>(p.src, row, col + 2 * i + 1).v[0];
      const float2 cs = rt[i];
      st(dst + 2 * i, x * cs.x - y * cs.y);
      st(dst + 2 * i + 1, y * cs.x + x * cs.y);
    }
  };
  if (u < p.heads) {
    T* plain = (T*)p.q_plain + ((size_t)row * p.heads + u) * p.plain_stride;
    for (int c = lane * VEC; c < p.dim; c += 32 * VEC) store_vec<VEC>(plain + c, mat_value<T, VEC>(p.src, row, u * per_head + c));
    for (int c = p.dim + lane; c < p.plain_stride; c += 32) st(plain + c, 0.f);
    T* q = (T*)p.q + ((size_t)row * p.heads + u) * a.L.kd;
    rotate(q + p.rank, u * per_head + p.dim);
    for (int c = a.L.key_dim + lane; c < a.L.kd; c += 32) st(q + c, 0.f);
    return;
  }
  const int pos = a.pos[row], seq = a.row_seq[row];
  const int page_idx = pos / a.d.page_size, slot = pos - page_idx * a.d.page_size;
  // a step whose reservation failed has no page for this row: nothing is written (the error word is set)
  if (seq < 0 || seq >= a.d.max_seqs || page_idx >= a.d.seq_pages[seq]) return;
  const int page = a.d.block_table[(size_t)seq * a.d.max_pages_per_seq + page_idx];
  T* dst = (T*)((char*)a.d.k_pool + a.L.k_off) + ((size_t)page * a.d.page_size + slot) * (size_t)a.L.kd;
  const int col = p.heads * per_head;
  float ss = 0.f;
  for (int c = lane * VEC; c < p.rank; c += 32 * VEC) {
    const Vec<VEC> v = mat_value<T, VEC>(p.src, row, col + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += v.v[e] * v.v[e];
  }
  const float r = 1.0f / sqrtf(warp_sum(ss) / (float)p.rank + p.eps);
  for (int c = lane * VEC; c < p.rank; c += 32 * VEC) {
    Vec<VEC> v = mat_value<T, VEC>(p.src, row, col + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] *= r * p.norm[c + e];
    store_vec<VEC>(dst + c, v);
  }
  rotate(dst + p.rank, col + p.rank);
}

}  // namespace

b200_status b200_rotation_table(const double* d_freq, int dims, const int32_t* d_pos, int rows, float2* d_out, void* stream) {
  if (rows <= 0 || dims < 2) return B200_OK;
  const long long n = (long long)rows * (dims / 2);
  rotation_table_kernel<<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(d_freq, dims / 2, d_pos, rows, d_out);
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
  const bool v4 = p.dim % 4 == 0 && p.rot % 4 == 0 && p.rank % 4 == 0 && p.plain_stride % 4 == 0 && (p.src.ws || p.src.y_stride % 4 == 0);
  auto* kernel = kv->dev.elem_bytes == 4 ? (v4 ? latent_prep_kernel<float, 4> : latent_prep_kernel<float, 1>)
                                         : (v4 ? latent_prep_kernel<__nv_bfloat16, 4> : latent_prep_kernel<__nv_bfloat16, 1>);
  kernel<<<dim3(rows, (p.heads + 1 + 7) / 8), 256, 0, (cudaStream_t)stream>>>(a);
  B200_LAUNCH_CHECK();
  return B200_OK;
}
