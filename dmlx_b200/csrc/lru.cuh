// Gated linear recurrent unit over the recurrent state of a layered pool (lru.cu).
#pragma once
#include "kv_pool.cuh"
#include "rows.cuh"
#include "short_conv.cuh"

// One layer over the rows of a step.  src columns [y | x], `width` each.  Prep: y -> gelu_tanh(y + y_bias) into out, and u = conv(x + x_bias)
// into `u` ([rows][blocks][u_group], zero behind a block's width).  Between the two the caller multiplies every block of u with its two
// gate matrices.  Scan: r = sigmoid(gate_r + r_bias), i = sigmoid(gate_i + i_bias), a = exp(-r * rate), S <- a S + sqrt(1 - a^2) i u, out *= S.
struct LruCall {
  int layer = 0, width = 0, blocks = 1;
  MatSrc src;
  const float *y_bias = nullptr, *x_bias = nullptr;  // [width]
  ShortConv conv;                // its state is set by the calls below: behind S in the slot's state
  void* u = nullptr;
  int u_group = 0;
  const float* gates = nullptr;  // [rows][blocks][r | i], a block's width each
  const float *r_bias = nullptr, *i_bias = nullptr, *rate = nullptr;  // [width]
  void* out = nullptr;
  int out_stride = 0;
};
constexpr int b200_lru_conv_off(int width) { return (width + 3) / 4 * 4; }
constexpr int b200_lru_elems(int width, int taps) { return b200_lru_conv_off(width) + (taps > 1 ? taps - 1 : 0) * width; }

b200_status b200_lru_prep(b200_kv* kv, LruCall c, const int32_t* d_cu, const int32_t* d_row_to_req, const int32_t* d_row_seq, const int32_t* d_pos,
                          int total_rows, void* stream);
b200_status b200_lru_scan(b200_kv* kv, const LruCall& c, const int32_t* d_cu, const int32_t* d_row_seq, const int32_t* d_pos, int n_req, int total_rows,
                          void* stream);
