// Attention over a span of the cache: the last `window` positions and the first `keep` ones, keys and values of
// different widths, one or two score maps per head over the same values, a rotated part behind queries and keys, values
// that are the front of the keys, a sink in the softmax, a gate per head (attn_span.cu).
#pragma once
#include "common.cuh"

struct SpanParams {
  // One row per token: [q: heads x maps x kd | k: groups x maps x kd | v: groups x vd] at these columns, f32.
  const float* qkv = nullptr;
  uint32_t ld = 0, k_off = 0, v_off = 0;
  const float *q_norm = nullptr, *k_norm = nullptr;  // [kd] RMS-norm weights per head and map, NULL: none
  float eps = 0.0f;
  uint32_t T = 0, G = 0, rep = 1, maps = 1, kd = 0, vd = 0;  // rep query heads per key / value head
  uint32_t kdp = 0, vdp = 0;                                // kd, vd rounded up to multiples of 4: rows of the cache
  uint32_t cap = 0, window = 0xFFFFFFFFu, keep = 0;
  float scale = 1.0f;
  float *kcache = nullptr, *vcache = nullptr;  // [B, G, cap, maps * kdp], [B, G, cap, vdp]
  const int32_t* len = nullptr;
  float* q = nullptr;                          // steps of several tokens: normed and rotated queries [B*T][heads * maps * kdp (+ rotp)]
  // One map only.  Behind the kd elements of a query or key come `rot` rotated ones (rotp: rounded up to 4): neighbouring
  // elements are a pair, table [position][rot / 2] holds cosine and sine.  A row of the cache is then kdp + rotp wide.
  uint32_t rot = 0, rotp = 0;
  const float2* table = nullptr;
  uint32_t q_step = 0, q_rot = 0, k_rot = 0;   // in qkv: floats between heads' queries (0: kd), where in a head the rotated part is; column of the keys'
  const float* q_main = nullptr;               // the queries' unrotated part, if it is not in qkv: [B*T][heads * kd]
  uint32_t qd = 0, qdp = 0;                    // ruai_span_append: width of the queries' unrotated part where it is not kd
  bool shared = false;                         // values are the first vd elements of the keys; no vcache
  const float* sink = nullptr;                 // [heads]: exp(sink) joins the softmax's denominator, once and unscaled
  const float* gate = nullptr;                 // [B*T, ld_gate]: factor of every head's output
  uint32_t ld_gate = 0;
  uint32_t out_step = 0;                       // floats between heads' outputs (0: vd)
  // two maps: the output is out_scale * rms_norm(map 1 - lambda map 2), over vd
  const float* lambda = nullptr;
  float out_scale = 1.0f;
  void* out = nullptr;
  uint32_t out_ld = 0;
  int out_dtype = RUAI_F32;
  float* scratch = nullptr;                    // key splits: see ruai_attn_span_scratch
  unsigned* counters = nullptr;                // zero between launches
  int* status = nullptr;
};
// Scratch (bytes, and zeroed counters) for the key splits of a step of T tokens over a cache of `cap` positions.
size_t ruai_attn_span_scratch(const SpanParams& p, uint32_t B, size_t* counters);
// One token: norms, append to the cache and attention in one kernel.  Several: norm and append, then attention (query
// tiles from eight tokens on where the shape allows it).
int ruai_attn_span(ruai_ctx* c, const SpanParams& p, uint32_t B);
// The first part of a step of several tokens alone: queries to p.q, keys and values to the cache.
int ruai_span_append(ruai_ctx* c, const SpanParams& p, uint32_t B);
// exp(sum a1 b1) - exp(sum a2 b2) + add, one number.
int ruai_diff_lambda(ruai_ctx* c, const float* a1, const float* b1, const float* a2, const float* b2, uint32_t n, float add, float* out);
