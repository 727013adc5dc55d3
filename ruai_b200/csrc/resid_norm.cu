// Norm of a sublayer's result, addition to the residual stream and the next sublayer's norm in one kernel (see
// resid_norm.cuh).  A CTA per row; the row stays in shared memory, every thread coming back to its own elements, so the
// only exchanges are the four sums.  The stream and the norms' weights are requested ahead of the dependency wait.
#include "resid_norm.cuh"

#include "vec.cuh"

namespace {

constexpr int kMaxThreads = 512;

template <int V> __device__ __forceinline__ Vec<V> ldv_or_zero(const float* p, uint32_t i) {
  if (p) return ldv<V>(p + i);
  Vec<V> r;
#pragma unroll
  for (int e = 0; e < V; ++e) r.f[e] = 0.0f;
  return r;
}
// Sum over the CTA; `red` holds a float per warp and is not used by the next sum but one.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  if (lane == 0) red[w] = v;
  __syncthreads();
  v = lane < nw ? red[lane] : 0.0f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  return v;
}

template <int V>
__global__ void __launch_bounds__(kMaxThreads) resid_norm_kernel(const ResidNormParams p) {
  extern __shared__ __align__(16) float row[];  // [d] the stream, [d] the sublayer's result
  __shared__ float red[2][32];
  float* ys = row + p.d;
  const uint32_t d = p.d, n = blockIdx.x, t0 = threadIdx.x * V, dt = blockDim.x * V;
  int flip = 0;
  // mean and 1 / deviation of the row in shared memory; every thread reads back what it wrote itself
  auto moments = [&](const float* v, bool center, float& mean, float& rs) {
    mean = 0.0f;
    if (center) {
      float s = 0.0f;
      for (uint32_t i = t0; i < d; i += dt) {
        const Vec<V> a = ldv<V>(v + i);
#pragma unroll
        for (int e = 0; e < V; ++e) s += a.f[e];
      }
      mean = block_sum(s, red[flip]) / (float)d;
      flip ^= 1;
    }
    float s = 0.0f;
    for (uint32_t i = t0; i < d; i += dt) {
      const Vec<V> a = ldv<V>(v + i);
#pragma unroll
      for (int e = 0; e < V; ++e) { const float q = a.f[e] - mean; s = fmaf(q, q, s); }
    }
    rs = 1.0f / sqrtf(block_sum(s, red[flip]) / (float)d + p.eps);
    flip ^= 1;
  };
  auto place = [&]() { return p.list ? (size_t)p.list[n] : p.step ? (size_t)(n + 1) * p.step - 1 : (size_t)n; };
  const bool early = p.x_early && !p.list;
  if (early) {
    const float* x = p.x + place() * d;
    for (uint32_t i = t0; i < d; i += dt) stv<V>(row, RUAI_F32, i, ldv<V>(x + i));
  }
  {
    auto fetch = [&](const float* q) { for (uint32_t i = t0; q && i < d; i += dt) asm volatile("prefetch.global.L2 [%0];" ::"l"(q + i)); };
    fetch(p.post.w); fetch(p.post.b); fetch(p.pre.w); fetch(p.pre.b);
  }
  grid_dependency_wait();
  grid_launch_dependents();
  const size_t at = place();
  if (!early) {
    const float* x = p.x + at * d;
    for (uint32_t i = t0; i < d; i += dt) stv<V>(row, RUAI_F32, i, ldv<V>(x + i));
  }
  if (p.post.w) {
    if (p.parts == 0) {
      const float* y = p.y + at * d;
      for (uint32_t i = t0; i < d; i += dt) stv<V>(ys, RUAI_F32, i, ldv<V>(y + i));
    } else {
      for (uint32_t i = t0; i < d; i += dt) {
        Vec<V> s;
#pragma unroll
        for (int e = 0; e < V; ++e) s.f[e] = 0.0f;
        for (uint32_t q = 0; q < p.parts; ++q) {
          const size_t o = at * p.parts + q;
          const float w = p.part_weight[o];
          const Vec<V> a = ldv<V>(p.y + (p.part_row ? (size_t)p.part_row[o] : o) * d + i);
#pragma unroll
          for (int e = 0; e < V; ++e) s.f[e] = fmaf(w, a.f[e], s.f[e]);
        }
        stv<V>(ys, RUAI_F32, i, s);
      }
    }
    float mean, rs;
    moments(ys, p.post.center, mean, rs);
    for (uint32_t i = t0; i < d; i += dt) {
      const Vec<V> w = ldv<V>(p.post.w + i), b = ldv_or_zero<V>(p.post.b, i), a = ldv<V>(ys + i);
      Vec<V> x = ldv<V>(row + i);
#pragma unroll
      for (int e = 0; e < V; ++e) x.f[e] += (a.f[e] - mean) * rs * w.f[e] + b.f[e];
      stv<V>(row, RUAI_F32, i, x);
      if (p.x_out) stv<V>(p.x_out, RUAI_F32, at * d + i, x);
    }
  }
  if (p.cat)
    for (uint32_t i = t0; i < d; i += dt) stv<V>(p.cat, p.dtype, (size_t)n * p.cat_ld + i, ldv<V>(row + i));
  if (p.pre.w) {
    float mean, rs;
    moments(row, p.pre.center, mean, rs);
    for (uint32_t i = t0; i < d; i += dt) {
      const Vec<V> w = ldv<V>(p.pre.w + i), b = ldv_or_zero<V>(p.pre.b, i);
      Vec<V> x = ldv<V>(row + i);
#pragma unroll
      for (int e = 0; e < V; ++e) x.f[e] = (x.f[e] - mean) * rs * w.f[e] + b.f[e];
      stv<V>(p.h, p.dtype, (size_t)n * p.h_ld + i, x);
    }
  }
}

__global__ void __launch_bounds__(256) embed_scaled_kernel(const int32_t* ids, const float* embed, float scale, uint32_t d, uint32_t vocab, float* x, void* copy,
                                                           uint32_t copy_ld, int dtype, int* err) {
  grid_dependency_wait();
  grid_launch_dependents();
  const uint32_t r = blockIdx.x;
  int32_t id = ids[r];
  if (id < 0 || (uint32_t)id >= vocab) {
    if (threadIdx.x == 0) atomicExch(err, 1);
    id = 0;
  }
  for (uint32_t i = threadIdx.x; i < d; i += blockDim.x) {
    const float v = embed[(size_t)id * d + i] * scale;
    x[(size_t)r * d + i] = v;
    if (copy) store_from_f32(copy, dtype, (size_t)r * copy_ld + i, v);
  }
}

}  // namespace

int ruai_resid_norm(ruai_ctx* c, const ResidNormParams& p) {
  if (p.rows == 0) return RUAI_OK;
  const size_t smem = 2 * (size_t)p.d * sizeof(float);
  if (smem > 200 * 1024) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "a residual stream of %u channels (at most 25600)", p.d);
  static bool attr_done[64] = {};
  if (!attr_done[c->ordinal & 63]) {
    RUAI_CUDA(c, cudaFuncSetAttribute(resid_norm_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    RUAI_CUDA(c, cudaFuncSetAttribute(resid_norm_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr_done[c->ordinal & 63] = true;
  }
  const bool v4 = p.d % 4 == 0 && (!p.h || p.h_ld % 4 == 0) && (!p.cat || p.cat_ld % 4 == 0);
  const uint32_t items = v4 ? p.d / 4 : p.d, most = p.rows >= 4u * 148u ? 256u : (uint32_t)kMaxThreads;
  const uint32_t threads = items >= most ? most : (items + 31) / 32 * 32;
  RUAI_CUDA(c, v4 ? ruai_launch(c, resid_norm_kernel<4>, dim3(p.rows), dim3(threads), smem, true, p)
                  : ruai_launch(c, resid_norm_kernel<1>, dim3(p.rows), dim3(threads), smem, true, p));
  return RUAI_OK;
}

int ruai_embed_scaled(ruai_ctx* c, const int32_t* ids, const float* embed, float scale, uint32_t rows, uint32_t d, uint32_t vocab, float* x, void* copy,
                      uint32_t copy_ld, int dtype, int* err) {
  RUAI_CUDA(c, ruai_launch(c, embed_scaled_kernel, dim3(rows), dim3(256), 0, true, ids, embed, scale, d, vocab, x, copy, copy_ld, dtype, err));
  return RUAI_OK;
}
