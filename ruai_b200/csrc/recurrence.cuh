// Linear attention with a matrix state per head and a per-channel decay (recurrence.cu).
#pragma once
#include "common.cuh"

// Per head, S [dk, dv] in f32:
//   bonus rule (u and k set):  o[c] = sum_i r[i] (S[i][c] + u[i] k[i] v[c]); afterwards S[i][c] <- w[i] S[i][c] + k[i] v[c]
//   otherwise (both NULL):     S[i][c] <- w[i] S[i][c] + (1 - w[i]) v[c]; afterwards o[c] = sum_i r[i] S[i][c]
// The state before the first token (*len == 0) is zero.
struct RecurrenceParams {
  const float *r = nullptr, *k = nullptr, *w = nullptr, *v = nullptr;  // rows of tokens, `ld*` apart; head h at column h * dk (v: h * dv)
  uint32_t ld_r = 0, ld_k = 0, ld_w = 0, ld_v = 0;
  // alternatively (single-token steps) w = exp(-exp(W t + w0)), W rows of `rank` elements (QL_DENSE layout), t [B, ld_t]
  const void* w2 = nullptr;
  int w2_bits = 16;
  const void* t = nullptr;
  int t_dtype = RUAI_F32;
  uint32_t rank = 0, w2_ld = 0, ld_t = 0;
  const float* w0 = nullptr;
  const float* u = nullptr;      // [H, dk]
  float* state = nullptr;        // [B, H, dk, dv]
  const int32_t* len = nullptr;
  uint32_t T = 0, H = 0, dk = 0, dv = 0;
  float* o = nullptr;            // [B*T, H * dv] raw outputs (steps of several tokens)
  // the head's output norm: o / rms(o) * norm (* gate)
  float eps = 0.0f;
  const float* norm = nullptr;   // [dv], or [H * dv] (norm_per_head)
  int norm_per_head = 0;
  const float* gate = nullptr;   // [B*T, ld_gate]
  uint32_t ld_gate = 0;
  void* out = nullptr;           // [B*T, out_ld]
  uint32_t out_ld = 0;
  int out_dtype = RUAI_F32;
};
// The whole step: T == 1 one kernel, otherwise the scan and the output norm.
int ruai_recurrence(ruai_ctx* c, const RecurrenceParams& p, uint32_t B);
// The output norm alone: rows of raw outputs p.o; of the other members only H, dv and those of the norm matter.
int ruai_head_norm(ruai_ctx* c, const RecurrenceParams& p, uint32_t rows);
