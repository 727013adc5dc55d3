// Routing of tokens to experts (see moe.cuh).  The experts themselves are dense.cu's Linears of blocks: with few tokens
// every (token, choice) pair reads its expert's weights, with many the pairs are sorted by expert and go through the tensor
// cores tile by tile; resid_norm.cu adds the weighted results up.
#include "moe.cuh"

namespace {

// A warp per row; a lane holds every 32nd expert's choice score.
template <int PER>
__global__ void __launch_bounds__(256) route_kernel(const float* logits, uint32_t parts, const float* correction, uint32_t rows, uint32_t experts, uint32_t top,
                                                    float scale, int32_t* chosen, float* weight) {
  const uint32_t lane = threadIdx.x & 31, row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  float corr[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) corr[i] = (correction && lane + 32 * i < experts) ? correction[lane + 32 * i] : 0.0f;
  grid_dependency_wait();
  grid_launch_dependents();
  if (row >= rows) return;
  float score[PER], choice[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    float z = 0.0f;
    const float* src = logits + (size_t)row * parts * experts + min(lane + 32 * i, experts - 1);
#pragma unroll 8
    for (uint32_t q = 0; q < parts; ++q) z += src[(size_t)q * experts];
    score[i] = 1.0f / (1.0f + expf(-z));
    choice[i] = score[i] + corr[i];
  }
  uint32_t taken = 0;  // bit i: this lane's expert i is chosen already
  for (uint32_t s = 0; s < top; ++s) {
    float best = -INFINITY;
    uint32_t at = 0xFFFFFFFFu;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (!(taken >> i & 1u) && lane + 32 * i < experts && (choice[i] > best || at == 0xFFFFFFFFu)) { best = choice[i]; at = lane + 32 * i; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float b = __shfl_xor_sync(0xFFFFFFFFu, best, o);
      const uint32_t a = __shfl_xor_sync(0xFFFFFFFFu, at, o);
      if (a != 0xFFFFFFFFu && (at == 0xFFFFFFFFu || b > best || (b == best && a < at))) { best = b; at = a; }
    }
    if (at == 0xFFFFFFFFu) at = 0;  // cannot happen: top <= experts
    if ((at & 31u) == lane) {  // the lane that holds it
      taken |= 1u << (at >> 5);
      float w = score[0];
#pragma unroll
      for (int i = 1; i < PER; ++i) w = (at >> 5) == (uint32_t)i ? score[i] : w;
      chosen[(size_t)row * top + s] = (int32_t)at;
      weight[(size_t)row * top + s] = w * scale;
    }
  }
}

// One CTA: counts, first places, then the pairs' places.
__global__ void __launch_bounds__(1024) route_sort_kernel(const int32_t* chosen, uint32_t pairs, uint32_t top, uint32_t experts, uint32_t tile, uint32_t tiles,
                                                          const RouteTiles r) {
  __shared__ uint32_t count[kRouteExpertsMax], next[kRouteExpertsMax];
  __shared__ uint32_t part[32];
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  grid_dependency_wait();
  grid_launch_dependents();
  if (tid < experts) count[tid] = 0;
  __syncthreads();
  for (uint32_t i = tid; i < pairs; i += 1024) atomicAdd(&count[chosen[i]], 1u);
  for (uint32_t i = tid; i < tiles; i += 1024) r.expert[i] = -1;
  for (uint32_t i = tid; i < tiles * tile; i += 1024) r.source[i] = -1;
  __syncthreads();
  // an expert per thread: its tiles, and those of the ones before it
  const uint32_t mine = tid < experts ? (count[tid] + tile - 1) / tile : 0;
  uint32_t sum = mine;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const uint32_t v = __shfl_up_sync(0xFFFFFFFFu, sum, o);
    if (lane >= (uint32_t)o) sum += v;
  }
  if (lane == 31) part[warp] = sum;
  __syncthreads();
  uint32_t before = sum - mine;
  for (uint32_t w = 0; w < warp; ++w) before += part[w];
  if (tid < experts) {
    next[tid] = before * tile;
    for (uint32_t i = 0; i < mine; ++i) r.expert[before + i] = (int32_t)tid;
  }
  __syncthreads();
  for (uint32_t i = tid; i < pairs; i += 1024) {
    const uint32_t at = atomicAdd(&next[chosen[i]], 1u);  // any order within an expert: its rows do not meet
    r.place[i] = (int32_t)at;
    r.source[at] = (int32_t)(i / top);
  }
}

__global__ void __launch_bounds__(128) route_gather_kernel(const uint4* x, const int32_t* source, uint32_t n16, uint4* y) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int32_t s = source[blockIdx.x];
  if (s < 0) return;
  for (uint32_t i = threadIdx.x; i < n16; i += blockDim.x) y[(size_t)blockIdx.x * n16 + i] = x[(size_t)s * n16 + i];
}

}  // namespace

int ruai_route(ruai_ctx* c, const float* logits, uint32_t parts, const float* correction, uint32_t rows, uint32_t experts, uint32_t top, float scale,
               int32_t* chosen, float* weight) {
  if (!experts || experts > kRouteExpertsMax || !top || top > kRouteTopMax || top > experts)
    return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "%u of %u experts (at most %u of %u)", top, experts, kRouteTopMax, kRouteExpertsMax);
  const uint32_t warps = rows >= 1024 ? 8 : 1;
  const dim3 grid((rows + warps - 1) / warps), block(warps * 32);
  RUAI_CUDA(c, experts <= 64    ? ruai_launch(c, route_kernel<2>, grid, block, 0, true, logits, parts, correction, rows, experts, top, scale, chosen, weight)
               : experts <= 256 ? ruai_launch(c, route_kernel<8>, grid, block, 0, true, logits, parts, correction, rows, experts, top, scale, chosen, weight)
                                : ruai_launch(c, route_kernel<32>, grid, block, 0, true, logits, parts, correction, rows, experts, top, scale, chosen, weight));
  return RUAI_OK;
}

int ruai_route_sort(ruai_ctx* c, const int32_t* chosen, uint32_t rows, uint32_t top, uint32_t experts, uint32_t tile, const RouteTiles& out) {
  RUAI_CUDA(c, ruai_launch(c, route_sort_kernel, dim3(1), dim3(1024), 0, true, chosen, rows * top, top, experts, tile,
                           ruai_route_tiles(rows * top, experts, tile), out));
  return RUAI_OK;
}

int ruai_route_gather(ruai_ctx* c, const void* x, const int32_t* source, uint32_t n, uint32_t bytes, void* y) {
  if (bytes % 16) return ruai_fail(c, RUAI_ERR_ARG, "rows of %u bytes", bytes);
  RUAI_CUDA(c, ruai_launch(c, route_gather_kernel, dim3(n), dim3(128), 0, true, (const uint4*)x, source, bytes / 16, (uint4*)y));
  return RUAI_OK;
}
