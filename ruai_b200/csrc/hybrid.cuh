// A decoder built from a list of layers, each with its own kind of token mixer (hybrid.cu).
#pragma once
#include <string>
#include <vector>

#include "model.cuh"

// A weight by its name in a checkpoint; rows x cols f32 while it is set, and how synthetic weights fill it.
struct HybridTensor {
  std::string name;
  uint64_t id = 0;
  size_t rows = 0, cols = 0;
  float synth_std = 0.0f, synth_fill = 0.0f;
};

int hybrid_create(ruai_model* m, const ruai_hybrid_config& cfg, const ruai_layer_config* layers);
void hybrid_destroy(ruai_model* m);
const std::vector<HybridTensor>& hybrid_tensors(const ruai_model* m);
const HybridTensor* hybrid_tensor(const ruai_model* m, uint64_t id);
const HybridTensor* hybrid_tensor_by_name(const ruai_model* m, const char* name);
// Kernel-ready weights in bf16 (bits 16; bf16 activations) or f32 (bits 32) from the f32 tensors set so far.
int hybrid_build(ruai_model* m, uint32_t bits);
// heads 0: the layer caches no keys and values.
void hybrid_cache_shape(const ruai_model* m, uint32_t run, uint32_t* heads, uint32_t* kw, uint32_t* vw);
// Tables for positions up to `positions`.
int hybrid_positions(ruai_model* m, uint32_t positions);
int hybrid_state_alloc(ruai_model* m, uint32_t B);
int hybrid_reserve(ruai_model* m, uint32_t rows, uint32_t out_rows, uint32_t B, uint32_t T);
int hybrid_issue(ruai_model* m, uint32_t B, uint32_t T, const HeadRows& head, bool want_argmax);
int hybrid_time_linears(ruai_model* m, uint32_t B, uint32_t iters, float* ms_total, uint32_t* launches, double* bytes_per_pass);
double hybrid_step_bytes(const ruai_model* m, uint32_t B, uint32_t len);
