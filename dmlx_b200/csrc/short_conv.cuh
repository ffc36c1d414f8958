// Causal convolution over the last few tokens, channel by channel, in front of a recurrence or of attention.  The inputs of the last
// taps - 1 tokens of a sequence are part of its slot's state (f32): entry e holds the one at distance e + 1 before the next token.
//
// The rows of a step are worked on side by side.  Rows with less than taps - 1 rows of their request before them in the step read the
// state, so the worker of a request's first row takes all of those, and brings the state up to date behind them: no other worker
// touches it.
#pragma once
#include "rows.cuh"

struct ShortConv {
  int taps = 0, channels = 0;   // taps 0: no convolution
  const __nv_bfloat16* w = nullptr;  // [taps][channels], the current token's last
  const float* bias = nullptr;  // [channels] on the result, may be null
  float* state = nullptr;       // of slot 0
  size_t slot_elems = 0;
};

// Rows a worker that starts at `row` takes: none, its own, or at a request's start as many as read the state.
__device__ __forceinline__ int conv_rows(const ShortConv& s, int j, int count) {
  if (s.taps < 2 || j >= s.taps - 1) return 1;
  return j == 0 ? min(s.taps - 1, count) : 0;
}

// Result at one row.  j: rows of its request before it in this step; value(row, channel): input of a row of the step.
template <int VEC, typename F>
__device__ __forceinline__ Vec<VEC> conv_value(const ShortConv& s, F value, int row, int j, int pos, int slot, int c) {
  Vec<VEC> acc{};
  if (s.bias) acc = load_vec<VEC>(s.bias + c);
  const float* state = s.state + (size_t)slot * s.slot_elems + c;
  for (int d = min(s.taps - 1, pos); d >= 0; --d) {
    const Vec<VEC> u = d <= j ? value(row - d, c) : load_vec<VEC>(state + (size_t)(d - j - 1) * s.channels);
    const Vec<VEC> w = load_vec<VEC>(s.w + (size_t)(s.taps - 1 - d) * s.channels + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc.v[e] = fmaf(w.v[e], u.v[e], acc.v[e]);
  }
  return acc;
}

// Results at R consecutive rows of one request that do not read the state (the first has TAPS - 1 rows before it in the step).  The
// weights and the inputs between the rows are read once.
template <int TAPS, int R, int VEC, typename F>
__device__ __forceinline__ void conv_values_inside(const ShortConv& s, F value, int row, int c, Vec<VEC> (&out)[R]) {
  Vec<VEC> u[TAPS - 1 + R], w[TAPS], bias{};
#pragma unroll
  for (int i = 0; i < TAPS - 1 + R; ++i) u[i] = value(row - (TAPS - 1) + i, c);
#pragma unroll
  for (int t = 0; t < TAPS; ++t) w[t] = load_vec<VEC>(s.w + (size_t)t * s.channels + c);
  if (s.bias) bias = load_vec<VEC>(s.bias + c);
#pragma unroll
  for (int r = 0; r < R; ++r) {
    out[r] = bias;
#pragma unroll
    for (int t = 0; t < TAPS; ++t) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) out[r].v[e] = fmaf(w[t].v[e], u[r + t].v[e], out[r].v[e]);
    }
  }
}

// State behind a request whose first row in the step is r0 (entries move up, so the far ones are written first).
template <int VEC, typename F>
__device__ __forceinline__ void conv_update(const ShortConv& s, F value, int r0, int count, int slot, int c) {
  float* state = s.state + (size_t)slot * s.slot_elems + c;
  for (int d = s.taps - 1; d >= 1; --d)
    store_vec<VEC>(state + (size_t)(d - 1) * s.channels, d <= count ? value(r0 + count - d, c) : load_vec<VEC>(state + (size_t)(d - count - 1) * s.channels));
}
