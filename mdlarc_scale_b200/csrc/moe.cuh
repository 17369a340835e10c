// Routing of tokens to experts: arguments and launchers; see moe.cu.
#pragma once
#include "common.cuh"

constexpr int MOE_MAX_EXPERTS = 256;
constexpr int MOE_MAX_TOP = 32;

struct MoeArgs {
  int rows, experts, top;
  const float* z;          // [rows][z_pitch] router logits; null: computed here from xn and w_router
  int z_pitch;
  const void* w_router;    // [>= experts][pitch] activation format
  int gran;                // an expert's slots are padded to a multiple of gran (128 or 256)
  int max_slots;
  int* count;              // [experts], zero on entry: tokens of each expert
  int* expert;             // [rows * top]
  int* rank;               // [rows * top] place among the expert's tokens
  float* weight;           // [rows * top]
  int* slot;               // [rows * top]
  float* slot_weight;      // [max_slots], 0 in padding slots
  int* tile_expert;        // [max_slots / 128] expert of every 128-slot tile
  int* n_tiles;            // 128-slot tiles in use
  const void* xn;          // [rows][pitch] activation format
  void* xs;                // [max_slots][pitch]: the rows of xn in slot order
  int pitch, fmt;
};

// slots a call of `rows` rows can need
int arcb_moe_max_slots(int rows, int experts, int top, int gran);
// few enough rows that the router's product is cheaper inside the routing kernel than as a launch of its own
bool arcb_moe_router_inside(int rows, int experts, int pitch, int fmt);
int arcb_launch_moe_route(const MoeArgs& a, cudaStream_t stream);
void arcb_count_launch(long long n);
