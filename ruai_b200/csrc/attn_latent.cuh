// Latent attention beside attn_span.cu and attn_prefill.cu: few queries in the absorbed form, tables of rotations, and latents
// as the input of a matrix product (attn_latent.cu).
#pragma once
#include <vector>

#include "attn_span.cuh"

// Rotations of `dims` elements in pairs (2i, 2i + 1) by position * base^(-2i / dims).  factor != 0: pairs that turn through
// the original context less often than `slow` times have their frequency divided by factor, those that turn more than `fast`
// times keep it, between the two it is interpolated linearly in the pair's number; cosine and sine are then multiplied by
// 0.1 ln(factor) + 1.  (Peng, Quesnelle, Fan, Shippole: "YaRN: Efficient Context Window Extension of Large Language Models".)
struct RotaryConfig {
  uint32_t rot = 0, dims = 0;  // the elements rot beyond dims stay as they are
  double base = 10000.0, factor = 0.0, original = 0.0, fast = 0.0, slow = 0.0;
  bool operator==(const RotaryConfig& o) const {
    return rot == o.rot && dims == o.dims && base == o.base && factor == o.factor && original == o.original && fast == o.fast && slow == o.slow;
  }
};
// Frequencies of the dims / 2 pairs, and the factor of their cosines and sines.
std::vector<double> ruai_rotary_frequencies(const RotaryConfig& r, double* scale);
// table [positions][rot / 2]; angles in f64 before the table's entries are rounded to f32.  freq: device, dims / 2.
int ruai_rotary_table(ruai_ctx* c, const double* freq, uint32_t pairs, uint32_t rot_pairs, uint32_t positions, double scale, float2* table);
// Rows 0 .. n - 1 of every sequence's cache [B][cap][kw], their first `rank` elements, to [B * n][ld] (zeros past rank).
int ruai_latent_rows(ruai_ctx* c, const float* cache, uint32_t B, uint32_t cap, uint32_t kw, uint32_t n, uint32_t rank, void* out, uint32_t ld, int out_dtype);

// The attention of a step of few tokens where keys and values are one row per position (SpanParams::shared), rows of up to
// 640 floats without a window.  The step's queries and rows are prepared as for ruai_attn_span (T == 1: by the kernel).
struct LatentProjection {  // every head's result through its rows of w: block_n rows per head, the first `rows` of them count
  const ruai_qweight* w = nullptr;
  uint32_t block_n = 0, rows = 0;
  void* out = nullptr;     // [B*T, out_ld], head h at column h * rows
  uint32_t out_ld = 0;
  int out_dtype = RUAI_F32;
};
bool ruai_attn_latent_takes(const SpanParams& p);
size_t ruai_attn_latent_scratch(const SpanParams& p, uint32_t B);
// Results to p.out, or with `o` through the projection to o->out instead.
int ruai_attn_latent(ruai_ctx* c, const SpanParams& p, uint32_t B, const LatentProjection* o);
