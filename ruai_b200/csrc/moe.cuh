// Mixture of experts: which experts a token uses, and the tokens of every expert side by side (moe.cu).
#pragma once
#include "common.cuh"

constexpr uint32_t kRouteTopMax = 32;     // experts per token
constexpr uint32_t kRouteExpertsMax = 1024;

// Per row: the `top` experts with the largest score + correction (correction NULL: score; of equal ones the lower number),
// in that order, and their scores times `scale` as weights.  A score is the sigmoid of the sum of `parts` numbers, parts
// [rows][parts][experts] (a router's matrix product may be cut into parts along its inputs).
int ruai_route(ruai_ctx* c, const float* logits, uint32_t parts, const float* correction, uint32_t rows, uint32_t experts, uint32_t top, float scale,
               int32_t* chosen /* [rows, top] */, float* weight /* [rows, top] */);

// The (row, choice) pairs sorted by expert, every expert's share rounded up to whole tiles of `tile` rows.
struct RouteTiles {
  int32_t* place = nullptr;   // [rows * top]: where a pair went
  int32_t* source = nullptr;  // [tiles * tile]: the row at a place, -1 where nothing is
  int32_t* expert = nullptr;  // [tiles]: the tile's expert, -1: none
};
// Tiles that can come up.
inline uint32_t ruai_route_tiles(uint32_t pairs, uint32_t experts, uint32_t tile) { return pairs / tile + (pairs < experts ? pairs : experts); }
int ruai_route_sort(ruai_ctx* c, const int32_t* chosen, uint32_t rows, uint32_t top, uint32_t experts, uint32_t tile, const RouteTiles& out);
// Row i of y is row source[i] of x; where that is negative nothing is written.  Rows of `bytes` bytes, a multiple of 16.
int ruai_route_gather(ruai_ctx* c, const void* x, const int32_t* source, uint32_t n, uint32_t bytes, void* y);
