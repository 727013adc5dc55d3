// The step between two sublayers whose results are normed before they join the residual stream (resid_norm.cu).
#pragma once
#include "common.cuh"

struct NormWeights {
  const float* w = nullptr;  // [d]
  const float* b = nullptr;  // [d] or NULL
  bool center = true;        // LayerNorm: deviations from the mean; false: RMSNorm
};
// Per row: x += post(y), where y is the last sublayer's result; then any of
//   h = pre(x)                  the next sublayer's input
//   cat[0 .. d) = x             the left half of a matrix product's input [x | ...]
// Either of post and pre may be missing (w NULL).  Norms are (x - mean) / sqrt(var + eps) * w + b.
struct ResidNormParams {
  const float* x = nullptr;       // [rows, d]
  float* x_out = nullptr;         // may be x itself; NULL: the stream is not needed any more
  bool x_early = false;           // x is older than the predecessor kernel's results
  // y: [rows, d]; with `parts`, y's row for row r is the sum of part_weight[r * parts + i] * (row part_row[r * parts + i] of y)
  const float* y = nullptr;
  uint32_t parts = 0;
  const float* part_weight = nullptr;
  const int32_t* part_row = nullptr;  // NULL: row r * parts + i
  NormWeights post, pre;
  float eps = 0.0f;
  uint32_t rows = 0, d = 0;
  // the rows to work on: `list` [rows], or with a step, rows step - 1, 2 step - 1, ... (0: all)
  const int32_t* list = nullptr;
  uint32_t step = 0;
  void* h = nullptr;
  uint32_t h_ld = 0;              // row i of h belongs to the i-th row worked on
  void* cat = nullptr;
  uint32_t cat_ld = 0;
  int dtype = RUAI_F32;           // of h and cat
};
int ruai_resid_norm(ruai_ctx* c, const ResidNormParams& p);

// x = scale * embed[id] (rows of d); with `copy`, also into rows copy_ld apart of `dtype`.
int ruai_embed_scaled(ruai_ctx* c, const int32_t* ids, const float* embed, float scale, uint32_t rows, uint32_t d, uint32_t vocab, float* x, void* copy,
                      uint32_t copy_ld, int dtype, int* err);
