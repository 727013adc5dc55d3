// RMSNorm (one gain per channel or one for all) with token shift and further interpolations with the previous token.
//
// One CTA takes a few consecutive tokens of one sequence: the rows' 1 / rms first, then a walk over the tokens with a
// thread per channel, which keeps the previous token's two values in registers.  What precedes the step comes from the
// per-sequence state; a step of several tokens leaves its last token's values in a second buffer (other CTAs may still
// be reading the first), which the caller copies over afterwards.
#include "token_mix.cuh"

#include "vec.cuh"

namespace {

constexpr int kThreads = 256, kTok = 4;

__device__ float block_sum_256(float v, float* red) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  __syncthreads();
  if (lane == 0) red[w] = v;
  __syncthreads();
  float t = 0.0f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) t += red[i];
  return t;
}

// grid (groups of `tok` tokens, sequences, slices of the channels): where there are few tokens several CTAs share a row's
// channels, each summing up the whole row
template <int V>
__global__ void __launch_bounds__(kThreads) token_mix_kernel(const TokenMixParams p, uint32_t tok) {
  __shared__ float red[32], rstd[kTok + 2];
  const uint32_t slice = (p.d + gridDim.z * kThreads * V - 1) / (gridDim.z * kThreads * V) * (kThreads * V);
  const uint32_t c0 = blockIdx.z * slice, c1 = min(p.d, c0 + slice);
  if (gridDim.z > 1) {  // constants and the state of earlier steps do not depend on the predecessor kernel: into the L2
    const uint32_t i = c0 + threadIdx.x * V;
    auto fetch = [&](const float* q) { if (q && i < c1) asm volatile("prefetch.global.L2 [%0];" ::"l"(q + i)); };
    fetch(p.shift);
    if (p.state) { fetch(p.state + (size_t)blockIdx.y * 2 * p.d); fetch(p.state + (size_t)blockIdx.y * 2 * p.d + p.d); }
#pragma unroll
    for (int q = 0; q < kMixMax; ++q) if (q < p.n_mix) fetch(p.mu[q]);
  }
  grid_dependency_wait();
  grid_launch_dependents();
  const uint32_t b = blockIdx.y, t0 = blockIdx.x * tok, t1 = min(p.T, t0 + tok), d = p.d;
  const bool hist = p.shift != nullptr || p.n_mix > 0;
  const int first = hist ? max((int)t0 - 2, 0) : (int)t0;
  auto row_of = [&](uint32_t t) { return p.rows ? (size_t)p.rows[b * p.T + t] : (size_t)b * p.T + t; };
  for (uint32_t t = (uint32_t)first; t < t1; ++t) {
    const float* xr = p.x + row_of(t) * d;
    float s = 0.0f;
#pragma unroll 4
    for (uint32_t i = threadIdx.x * V; i < d; i += kThreads * V) {
      const Vec<V> v = ldv<V>(xr + i);
#pragma unroll
      for (int e = 0; e < V; ++e) s = fmaf(v.f[e], v.f[e], s);
    }
    s = block_sum_256(s, red);
    if (threadIdx.x == 0) rstd[t - (uint32_t)first] = 1.0f / sqrtf(s / (float)d + p.eps);
  }
  __syncthreads();
  const bool fresh = hist && *p.len == 0;  // nothing precedes the sequence's first token
  for (uint32_t i = c0 + threadIdx.x * V; i < c1; i += kThreads * V) {
    Vec<V> g, sh, h1, s1;
    if (p.g_vec) g = ldv<V>(p.g + i);
    else {
#pragma unroll
      for (int e = 0; e < V; ++e) g.f[e] = *p.g;
    }
#pragma unroll
    for (int e = 0; e < V; ++e) { sh.f[e] = 0.0f; h1.f[e] = 0.0f; s1.f[e] = 0.0f; }
    auto h_of = [&](uint32_t t) {
      Vec<V> v = ldv<V>(p.x + row_of(t) * d + i);
      const float r = rstd[t - (uint32_t)first];
#pragma unroll
      for (int e = 0; e < V; ++e) v.f[e] = v.f[e] * r * g.f[e];
      return v;
    };
    if (hist) {
      if (p.shift) sh = ldv<V>(p.shift + i);
      const float* st = p.state + (size_t)b * 2 * d + i;
      if (t0 == 0) {
        if (!fresh) { h1 = ldv<V>(st); s1 = ldv<V>(st + d); }
      } else {
        Vec<V> h2;
#pragma unroll
        for (int e = 0; e < V; ++e) h2.f[e] = 0.0f;
        if (t0 >= 2) h2 = h_of(t0 - 2);
        else if (!fresh) h2 = ldv<V>(st);
        h1 = h_of(t0 - 1);
#pragma unroll
        for (int e = 0; e < V; ++e) s1.f[e] = h1.f[e] + (h2.f[e] - h1.f[e]) * sh.f[e];
      }
    }
    for (uint32_t t = t0; t < t1; ++t) {
      const Vec<V> h = h_of(t);
      Vec<V> s;
#pragma unroll
      for (int e = 0; e < V; ++e) s.f[e] = h.f[e] + (h1.f[e] - h.f[e]) * sh.f[e];
      const size_t o = ((size_t)b * p.T + t) * p.ld + i;
      if (p.h_out) stv<V>(p.h_out, p.out_dtype, o, h);
      if (p.n_mix == 0) {
        if (p.mix_out[0]) stv<V>(p.mix_out[0], p.out_dtype, o, s);
      } else {
#pragma unroll
        for (int q = 0; q < kMixMax; ++q) {
          if (q < p.n_mix) {
            const Vec<V> mu = ldv<V>(p.mu[q] + i);
            Vec<V> y;
#pragma unroll
            for (int e = 0; e < V; ++e) y.f[e] = s.f[e] + (s1.f[e] - s.f[e]) * mu.f[e];
            stv<V>(p.mix_out[q], p.out_dtype, o, y);
          }
        }
      }
      h1 = h; s1 = s;
    }
    if (hist && p.state_out && t1 == p.T) {
      float* st = p.state_out + (size_t)b * 2 * d + i;
      stv<V>(st, RUAI_F32, 0, h1);
      stv<V>(st, RUAI_F32, d, s1);
    }
  }
}

}  // namespace

int ruai_token_mix(ruai_ctx* c, const TokenMixParams& p, uint32_t B) {
  if (p.n_mix > kMixMax) return ruai_fail(c, RUAI_ERR_ARG, "%d interpolations (at most %d)", p.n_mix, kMixMax);
  // several tokens per CTA once there are CTAs enough: the overlap of two rows costs less then
  const uint32_t tok = (size_t)B * p.T >= 4u * 148u ? kTok : 1u;
  const bool v4 = p.d % 4 == 0 && p.ld % 4 == 0;
  const uint32_t per = kThreads * (v4 ? 4u : 1u), most = (p.d + per - 1) / per, ctas = (p.T + tok - 1) / tok * B;
  const uint32_t slices = ctas >= 148u ? 1u : (148u / ctas < most ? 148u / ctas : most);
  const dim3 grid((p.T + tok - 1) / tok, B, slices);
  RUAI_CUDA(c, v4 ? ruai_launch(c, token_mix_kernel<4>, grid, dim3(kThreads), 0, true, p, tok)
                  : ruai_launch(c, token_mix_kernel<1>, grid, dim3(kThreads), 0, true, p, tok));
  return RUAI_OK;
}
