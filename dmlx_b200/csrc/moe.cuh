// Experts of a decoder layer (moe.cu): chosen by token id, the plan of a step for all layers at once, or by a router.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "dmlx_b200.h"
#include "rows.cuh"

// One layer on the device: its table [vocab][top] (null with a router) and where the plan goes, for up to max_rows * top assignments.
struct MoeTableLayer {
  const int* table = nullptr;
  int n_experts = 0, top = 0;
  uint32_t* indices = nullptr;  // expert of every assignment (token * top + place)
  int *offsets = nullptr, *order = nullptr, *inv_order = nullptr, *n_items = nullptr;
  int4* items = nullptr;        // {expert, first sorted row, rows}
};
int b200_moe_max_experts();
// Limits of a layer's router.
int b200_moe_max_top();
int b200_moe_max_groups();
b200_status b200_moe_table_plan(const MoeTableLayer* d_layers, int n_layers, int most_experts, const uint32_t* d_tokens, int n_tokens, int vocab,
                                int tile_rows, void* stream);
// Weights of the chosen experts: their softmax scores, divided by the sum of them (or not), times scale.  shared: where the sigmoid of one
// more logit behind the experts' goes, the weight of a token's shared expert.
struct RouterScores {
  bool renormalise = true;
  float scale = 1.f;
  float* shared = nullptr;
};
// Routes the tokens of one layer by their router logits (softmax, best experts of the best keep_groups of n_groups groups) and plans its
// matmuls.  f32: how logits that the matmul wrote itself are stored.
b200_status b200_moe_route_plan(const MoeTableLayer& L, const MatSrc& logits, bool f32, int n_groups, int keep_groups, int n_tokens, int tile_rows,
                                float* d_weights, void* stream, const RouterScores& scores = RouterScores{});
// out[p] = x[order[p] / top], bf16 rows of `width` elements (a multiple of 8).
b200_status b200_moe_gather_order(const void* d_x, const int* d_order, int top, int n_assign, int width, void* d_out, void* stream);
