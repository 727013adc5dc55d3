// Gated delta rule: a matrix state per head that corrects what it answers to a key, behind short convolutions (delta.cu).
#pragma once
#include "common.cuh"

constexpr int kConvMax = 16;  // taps of the convolutions

// Raw projections, f32 rows of tokens: q and k [G * dk] (kv head g at column g * dk), v [H * dv].  Each channel goes through
// a causal convolution over its last `taps` values (the newest with the last weight) and silu; q and k are made unit vectors
// per head (x / sqrt(sum x^2 + unit_eps)), q is then multiplied by q_scale.  Head h uses the q and k of kv head h / (H / G).
//   decay = exp(-exp(a_log[h]) softplus(a)), a with its bias added; beta as it is
//   S <- decay S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// and the output is o / rms(o) * norm * gate.  Before the first token (*len == 0) state and convolution inputs are zero.
struct DeltaParams {
  const float *q = nullptr, *k = nullptr, *v = nullptr, *a = nullptr, *beta = nullptr;
  uint32_t ld_q = 0, ld_k = 0, ld_v = 0, ld_a = 0, ld_beta = 0;
  const float *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr;  // [channels, taps]
  uint32_t taps = 1;
  float unit_eps = 1e-6f, q_scale = 1.0f;
  const float* a_log = nullptr;   // [H]
  float* state = nullptr;         // [B, H, dk, dv]
  float* history = nullptr;       // [B, taps, 2 G dk + H dv]: the projections (q | k | v) of position p in slot p mod taps
  const int32_t* len = nullptr;
  uint32_t T = 0, H = 0, G = 0, dk = 0, dv = 0;
  float eps = 0.0f;
  const float* norm = nullptr;    // [dv]
  const float* gate = nullptr;    // [B*T, ld_gate]
  uint32_t ld_gate = 0;
  void* out = nullptr;            // [B*T, out_ld]
  uint32_t out_ld = 0;
  int out_dtype = RUAI_F32;
  float* work = nullptr;          // steps of several tokens: ruai_delta_work floats
};
// For up to `rows` tokens of up to B sequences.
size_t ruai_delta_work(const DeltaParams& p, uint32_t rows, uint32_t B);
// The whole step: T == 1 one kernel, otherwise convolution, scan and output norm.
int ruai_delta(ruai_ctx* c, const DeltaParams& p, uint32_t B);
