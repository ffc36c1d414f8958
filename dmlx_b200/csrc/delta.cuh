// Gated delta rule over the recurrent state of a layered pool (delta.cu).
#pragma once
#include "gla.cuh"
#include "kv_pool.cuh"
#include "rows.cuh"
#include "short_conv.cuh"

// One layer over the rows of a step.  src columns [q | k | v | g | b | a] of widths kv_heads * dk, kv_heads * dk, heads * dv, heads * dv, heads,
// heads.  q, k and v pass a short convolution and silu; q and k of a head become unit vectors (kDeltaUnitEps inside the root), q also times
// dk^(-1/2).  Per head h with the q and k of head h / (heads / kv_heads): decay e^(-rate softplus(a + dt_bias)), beta = sigmoid(b),
// S <- decay S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q; the output row is rms_norm(o) * norm * silu(g), [heads][dv].
struct DeltaCall {
  int layer = 0, heads = 0, kv_heads = 0, dk = 0, dv = 0;
  MatSrc src;
  ShortConv conv;                                // taps and weights; its state is set by b200_delta_run
  const float *rate = nullptr, *dt_bias = nullptr;  // [heads]
  const float* norm = nullptr;                   // [dv]
  float eps = 0.f;
  void* out = nullptr;
  int out_stride = 0;
};
constexpr float kDeltaUnitEps = 1e-6f;
// A slot's state: S [heads][dk][dv], then the convolution's inputs.
constexpr int b200_delta_conv_off(int heads, int dk, int dv) { return (heads * dk * dv + 3) / 4 * 4; }
constexpr int b200_delta_channels(int heads, int kv_heads, int dk, int dv) { return 2 * kv_heads * dk + heads * dv; }
constexpr int b200_delta_elems(int heads, int kv_heads, int dk, int dv, int taps) {
  return b200_delta_conv_off(heads, dk, dv) + (taps > 1 ? taps - 1 : 0) * b200_delta_channels(heads, kv_heads, dk, dv);
}
// In front of the recurrence (convolutions, unit vectors, gates), and the recurrence itself with norm and output gate.
b200_status b200_delta_prep(b200_kv* kv, const GlaScratch& g, const DeltaCall& c, const int32_t* d_cu, const int32_t* d_row_to_req,
                            const int32_t* d_row_seq, const int32_t* d_pos, int total_rows, void* stream);
b200_status b200_delta_run(b200_kv* kv, const GlaScratch& g, const DeltaCall& c, const int32_t* d_cu, const int32_t* d_row_seq, const int32_t* d_pos,
                           int n_req, int total_rows, bool chunked, void* stream);
