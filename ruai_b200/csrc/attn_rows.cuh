// Queries and keys on their way to the cache: norm and rotation, a warp per row (attn_span.cu, attn_latent.cu).
#pragma once
#include "attn_span.cuh"

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xFFFFFFFFu, v, o));
  return v;
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }
// One warp: dst[0 .. n) = src * rstd * w (w NULL: src), zeros up to np.
__device__ __forceinline__ void norm_row(const float* src, const float* w, float eps, uint32_t n, uint32_t np, float* dst, uint32_t lane) {
  float rs = 1.0f;
  if (w) {
    float ss = 0.0f;
    for (uint32_t e = lane; e < n; e += 32) ss = fmaf(src[e], src[e], ss);
    ss = warp_sum(ss);
    rs = 1.0f / sqrtf(ss / (float)n + eps);
  }
  for (uint32_t e = lane; e < np; e += 32) dst[e] = e < n ? (w ? src[e] * rs * w[e] : src[e]) : 0.0f;
}

// One warp: the rotated part of a query or key, dst[0 .. rot), zeros up to rotp.
__device__ __forceinline__ void rotate_row(const float* src, const float2* cs, uint32_t rot, uint32_t rotp, float* dst, uint32_t lane) {
  for (uint32_t i = lane; i < rotp / 2; i += 32) {
    float u = 2 * i < rot ? src[2 * i] : 0.0f, v = 0.0f;
    if (2 * i + 1 < rot) {
      v = src[2 * i + 1];
      const float2 t = cs[i];
      const float w = u;
      u = fmaf(w, t.x, -(v * t.y));
      v = fmaf(v, t.x, w * t.y);
    }
    dst[2 * i] = u;
    dst[2 * i + 1] = v;
  }
}
// One warp: query e of a token (heads and maps), and the key of a group and map.
__device__ __forceinline__ void query_row(const SpanParams& p, size_t token, const float* row, uint32_t e, uint32_t nq, uint32_t pos, float* dst, uint32_t lane) {
  const uint32_t d = p.qd ? p.qd : p.kd, dp = p.qd ? p.qdp : p.kdp;
  const float* src = row + (size_t)e * (p.q_step ? p.q_step : d);
  norm_row(p.q_main ? p.q_main + (token * nq + e) * d : src, p.q_norm, p.eps, d, dp, dst, lane);
  if (p.rot) rotate_row(src + p.q_rot, p.table + (size_t)pos * (p.rot / 2), p.rot, p.rotp, dst + dp, lane);
}
__device__ __forceinline__ void key_row(const SpanParams& p, const float* row, uint32_t e, uint32_t pos, float* dst, uint32_t lane) {
  norm_row(row + p.k_off + (size_t)e * p.kd, p.k_norm, p.eps, p.kd, p.kdp, dst, lane);
  if (p.rot) rotate_row(row + p.k_rot, p.table + (size_t)pos * (p.rot / 2), p.rot, p.rotp, dst + p.kdp, lane);
}
