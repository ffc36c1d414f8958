// Latent attention over one layer of a layered pool whose values lie inside its key rows (attn_latent.cu).
#pragma once
#include "kv_pool.cuh"
#include "rows.cuh"

// Cosine and sine of every row's rotation times `size`, [rows][dims / 2]; made once per step for the layers that share frequencies.
b200_status b200_rotation_table(const double* d_freq, int dims, double size, const int32_t* d_pos, int rows, float2* d_out, void* stream);

// From the projection rows [heads x (dim + rot) | rank + rot] to what attention reads: the unrotated query parts ([heads][plain_stride],
// zero behind dim), the rotated ones (written at column `rank` of every head of q), and the normed latent with the rotated key
// part in its page.  Where the queries come out of a latent of their own (q_rank), one call takes [q_rank | rank + rot] and writes
// the normed query latent beside the page (heads = 0), and another takes the queries (keys = false).
struct LatentPrep {
  int layer = 0, heads = 0, dim = 0, rot = 0, rank = 0;
  bool halves = false;          // pairs are (i, i + rot / 2) instead of (2i, 2i + 1)
  bool keys = true;
  int q_rank = 0;
  const float* q_norm = nullptr;  // [q_rank]
  void* q_latent = nullptr;       // [rows][q_latent_stride], zero behind q_rank
  int q_latent_stride = 0;
  MatSrc src;
  const float* norm = nullptr;  // [rank]
  float eps = 0.f;
  const float2* rotation = nullptr;
  void* q_plain = nullptr;      // [rows][heads][plain_stride]
  int plain_stride = 0;
  void* q = nullptr;            // [rows][heads][stored key width]
};
b200_status b200_latent_prep(b200_kv* kv, const LatentPrep& p, const int32_t* d_pos, const int32_t* d_row_seq, int rows, void* stream);

// The tensor-core kernel (b200_window_attn_plan / _run come here for layers whose values lie in their keys).
bool b200_latent_attn_takes_mma(const b200_kv* kv, int32_t layer);
b200_status b200_latent_attn_plan(b200_kv* kv, int32_t layer, int32_t window, int32_t n_q_heads, const int32_t* d_row_seq, const int32_t* d_row_ctx, int32_t total_rows,
                                  void* stream);
b200_status b200_latent_attn_run(b200_kv* kv, const WindowAttnCall& c, const int32_t* d_row_seq, const int32_t* d_row_ctx, int32_t total_rows,
                                 void* stream);
