// RMSNorm followed by interpolations with the previous token (token_mix.cu).
#pragma once
#include "common.cuh"

constexpr int kMixMax = 6;

// Per token t: h[t] = g x[t] / rms(x[t]).  With a shift, s[t] = lerp(h[t], h[t - 1], shift), channel by channel; without,
// s = h.  Outputs: h itself (h_out, optional) and either s (n_mix == 0, if mix_out[0] is set) or n_mix interpolations
// lerp(s[t], s[t - 1], mu[i]).  Tokens of a step follow one another per sequence; what came before
// the step's first token is the state [B][2][d] (h and s of the last token), zero when *len is 0.
struct TokenMixParams {
  const float* x = nullptr;      // [B*T, d]
  const int32_t* rows = nullptr; // optional: row r of the outputs is row rows[r] of x (only without shift and mixes)
  const float* g = nullptr;      // [d], or one number (g_vec 0)
  int g_vec = 0;
  float eps = 0.0f;
  uint32_t T = 0, d = 0;
  const int32_t* len = nullptr;
  const float* shift = nullptr;  // [d] or NULL
  const float* state = nullptr;
  float* state_out = nullptr;    // may be `state` itself when T == 1
  void* h_out = nullptr;
  void* mix_out[kMixMax] = {};
  const float* mu[kMixMax] = {};
  int n_mix = 0;
  uint32_t ld = 0;               // row stride of every output
  int out_dtype = RUAI_F32;
};
int ruai_token_mix(ruai_ctx* c, const TokenMixParams& p, uint32_t B);
