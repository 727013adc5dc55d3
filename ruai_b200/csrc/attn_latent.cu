// Rotation tables and latent rows (see attn_latent.cuh).
#include "attn_latent.cuh"

#include <algorithm>
#include <cmath>

namespace {

__global__ void rotary_table_kernel(const double* freq, uint32_t pairs, uint32_t rot_pairs, uint32_t positions, double scale, float2* table) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)positions * rot_pairs) return;
  const uint32_t e = (uint32_t)(i % rot_pairs);
  double s = 0.0, c = 1.0;
  if (e < pairs) {
    sincos((double)(i / rot_pairs) * freq[e], &s, &c);
    s *= scale;
    c *= scale;
  }
  table[i] = make_float2((float)c, (float)s);
}

// grid (rows of a sequence, sequences)
__global__ void __launch_bounds__(128) latent_rows_kernel(const float* cache, uint32_t cap, uint32_t kw, uint32_t rank, void* out, uint32_t ld, int out_dtype) {
  grid_dependency_wait();
  grid_launch_dependents();
  const float* src = cache + ((size_t)blockIdx.y * cap + blockIdx.x) * kw;
  const size_t dst = ((size_t)blockIdx.y * gridDim.x + blockIdx.x) * ld;
  for (uint32_t e = threadIdx.x; e < ld; e += blockDim.x) store_from_f32(out, out_dtype, dst + e, e < rank ? src[e] : 0.0f);
}

}  // namespace

std::vector<double> ruai_rotary_frequencies(const RotaryConfig& r, double* scale) {
  std::vector<double> f(r.dims / 2);
  for (size_t i = 0; i < f.size(); ++i) f[i] = std::pow(r.base, -2.0 * (double)i / r.dims);
  *scale = 1.0;
  if (r.factor == 0.0) return f;
  const double two_pi = 6.283185307179586;
  // the pair (as a real number) that makes t turns within the original context
  auto pair_of = [&](double t) { return r.dims * std::log(r.original / (two_pi * t)) / (2.0 * std::log(r.base)); };
  const double lo = std::max(std::floor(pair_of(r.fast)), 0.0), hi = std::min(std::ceil(pair_of(r.slow)), r.dims - 1.0);
  for (size_t i = 0; i < f.size(); ++i) {
    const double ramp = std::min(std::max(((double)i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
    f[i] = f[i] / r.factor * ramp + f[i] * (1.0 - ramp);
  }
  *scale = 0.1 * std::log(r.factor) + 1.0;
  return f;
}

int ruai_rotary_table(ruai_ctx* c, const double* freq, uint32_t pairs, uint32_t rot_pairs, uint32_t positions, double scale, float2* table) {
  const size_t n = (size_t)positions * rot_pairs;
  if (n == 0) return RUAI_OK;
  rotary_table_kernel<<<(unsigned)((n + 255) / 256), 256, 0, c->stream>>>(freq, pairs, rot_pairs, positions, scale, table);
  RUAI_CUDA(c, cudaGetLastError());
  return RUAI_OK;
}

int ruai_latent_rows(ruai_ctx* c, const float* cache, uint32_t B, uint32_t cap, uint32_t kw, uint32_t n, uint32_t rank, void* out, uint32_t ld, int out_dtype) {
  if (B > 65535) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "%u sequences", B);
  RUAI_CUDA(c, ruai_launch(c, latent_rows_kernel, dim3(n, B), dim3(128), 0, true, cache, cap, kw, rank, out, ld, out_dtype));
  return RUAI_OK;
}
