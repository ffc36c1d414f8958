// Experts chosen by token id (moe.cu): the plan of a step for all layers at once.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "dmlx_b200.h"

// One layer on the device: its table [vocab][top] and where the plan goes, for up to max_rows * top assignments.
struct MoeTableLayer {
  const int* table = nullptr;
  int n_experts = 0, top = 0;
  uint32_t* indices = nullptr;  // expert of every assignment (token * top + place)
  int *offsets = nullptr, *order = nullptr, *inv_order = nullptr, *n_items = nullptr;
  int4* items = nullptr;        // {expert, first sorted row, rows}
};
int b200_moe_max_experts();
int b200_moe_max_top();
b200_status b200_moe_table_plan(const MoeTableLayer* d_layers, int n_layers, int most_experts, const uint32_t* d_tokens, int n_tokens, int vocab,
                                int tile_rows, void* stream);
// out[p] = x[order[p] / top], bf16 rows of `width` elements (a multiple of 8).
b200_status b200_moe_gather_order(const void* d_x, const int* d_order, int top, int n_assign, int width, void* d_out, void* stream);
