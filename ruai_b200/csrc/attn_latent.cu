// Latent attention of few queries, rotation tables and latent rows (see attn_latent.cuh).
//
// latent_attention_kernel: a CTA owns four heads of one query position and a share of the cached positions, which come into
// shared memory 64 at a time by bulk copies and serve as keys and as values.  Scores: a warp per two positions as they
// arrive, its lanes across the row, the four queries in registers, so that a row is read once; sums of values: a thread per
// four elements of the row and a group of the positions, all four heads in registers.  In the single-token step the kernel
// also rotates the queries, norms and rotates the new position's row and appends it; cached rows are requested ahead of the
// dependency wait.  Everything is f32.
//
// The shares' sums are merged by latent_project_kernel on their way through the values' projection, or, with more tokens than
// that reads its weights for, by latent_merge_kernel.
#include "attn_rows.cuh"

#include <algorithm>
#include <cmath>

#include "attn_latent.cuh"
#include "pipeline.cuh"

namespace {

using namespace pipe;

constexpr int kThreads = 256, kWarps = kThreads / 32, kHeads = 4, kPos = 64;
constexpr int kPart = 2 * kWarps, kParts = kPos / kPart;  // positions the warps score at a time, with a copy of their own
constexpr uint32_t kShares = 32;  // at most: a lane per share when they are merged

__device__ __forceinline__ float dot4(float4 a, float4 b, float s) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, s)))); }

// grid (sequences x groups of kHeads heads, T, shares); NE: four-element pieces of a row per lane, NV: of a value per thread
template <bool FUSE, int NE, int NV>
__global__ void __launch_bounds__(kThreads) latent_attention_kernel(const SpanParams p, uint32_t subs) {
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(16) float ps[kHeads][kPos];
  __shared__ float mr[kHeads], lr[kHeads], cr[kHeads];
  __shared__ __align__(8) uint64_t full[kParts];
  __shared__ int s_abort;
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t b = blockIdx.x / subs, head0 = blockIdx.x % subs * kHeads, t = blockIdx.y, share = blockIdx.z, shares = gridDim.z, H = p.rep;
  const uint32_t nh = min((uint32_t)kHeads, H - head0), kw = p.kdp + p.rotp, w4 = kw / 4, v4 = p.vdp / 4;
  float* ks = sm;  // [kPos][kw]
  float* base = p.kcache + (size_t)b * p.cap * kw;
  uint32_t pos = 0, i0 = 0, i1 = 0;
  bool over = false;
  auto plan = [&]() {
    pos = (uint32_t)__ldcg(p.len) + t;
    over = pos >= p.cap;  // the host grows the cache ahead of the step: touch nothing beyond it, tell the host
    const uint32_t n = pos + 1, per = (n + shares - 1) / shares;
    i0 = over ? 0 : min(n, share * per);
    i1 = over ? 0 : min(n, i0 + per);
  };
  // rows a .. e - 1 that are in the cache already; `coming`: how many of them
  uint32_t coming = 0;
  auto fetch = [&](uint32_t a, uint32_t e) {
    const uint32_t end = FUSE ? min(e, pos) : e;
    coming = end > a ? end - a : 0;
    if (tid == 0)
      for (uint32_t i = 0; i * kPart < coming; ++i) {
        const uint32_t n = min((uint32_t)kPart, coming - i * kPart);
        mbar_expect_tx(&full[i], n * kw * 4u);
        bulk_load(ks + (size_t)i * kPart * kw, base + (size_t)(a + i * kPart) * kw, n * kw * 4u, &full[i]);
      }
  };
  if (tid == 0) {
    for (int i = 0; i < kParts; ++i) mbar_init(&full[i], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    s_abort = 0;
  }
  if (FUSE) {  // cached rows and the position word are earlier steps' work
    plan();
    fetch(i0, min(i1, i0 + kPos));
  }
  grid_dependency_wait();
  grid_launch_dependents();
  if (!FUSE) {
    plan();
    fetch(i0, min(i1, i0 + kPos));
  }
  if (over && tid == 0 && p.status) atomicCAS(p.status, 0, 5);
  const size_t token = (size_t)b * p.T + t;
  const float* row = p.qkv + token * p.ld;
  // ---- this lane's pieces of the queries: all requested together, then rotated ----
  float4 q[kHeads][NE];
#pragma unroll
  for (int j = 0; j < NE; ++j) {
    const uint32_t f = lane + 32 * j;
    const bool main = 4 * f < p.kdp;
    const float* src = !FUSE ? p.q + (token * H + head0) * kw + 4 * f
                             : main ? p.q_main + (token * H + head0) * p.kd + 4 * f : row + (size_t)head0 * p.q_step + p.q_rot + 4 * f - p.kdp;
    const size_t step = !FUSE ? kw : main ? p.kd : p.q_step;
#pragma unroll
    for (int h = 0; h < kHeads; ++h)
      q[h][j] = (uint32_t)h < nh && f < w4 && !over ? *reinterpret_cast<const float4*>(src + h * step) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (FUSE && p.rot && !over) {
    const uint32_t pairs = p.rot / 2;
    const float2* cs = p.table + (size_t)pos * pairs;
#pragma unroll
    for (int j = 0; j < NE; ++j) {
      const uint32_t f = lane + 32 * j, i = 2 * f - p.kdp / 2;
      if (4 * f < p.kdp || f >= w4) continue;
      // two pairs; past the rotated ones the projection holds zeros
      const float2 c0 = i < pairs ? cs[i] : make_float2(1.f, 0.f), c1 = i + 1 < pairs ? cs[i + 1] : make_float2(1.f, 0.f);
#pragma unroll
      for (int h = 0; h < kHeads; ++h) {
        const float4 u = q[h][j];
        q[h][j] = make_float4(fmaf(u.x, c0.x, -(u.y * c0.y)), fmaf(u.y, c0.x, u.x * c0.y), fmaf(u.z, c1.x, -(u.w * c1.y)), fmaf(u.w, c1.x, u.z * c1.y));
      }
    }
  }
  if (tid < kHeads) {  // the sink is a first term without a value, in one of the shares
    const bool sink_here = p.sink && share == 0 && tid < nh;
    mr[tid] = sink_here ? p.sink[head0 + tid] : -INFINITY;
    lr[tid] = sink_here ? 1.0f : 0.0f;
  }
  // values: column pieces of a thread, and its group of the positions
  const uint32_t vcols = v4 > 64 ? 128u : v4 > 32 ? 64u : 32u, groups = kThreads / vcols, grp = tid / vcols, col = tid % vcols, per_group = kPos / groups;
  float4 acc[kHeads][NV];
#pragma unroll
  for (int h = 0; h < kHeads; ++h)
#pragma unroll
    for (int j = 0; j < NV; ++j) acc[h][j] = make_float4(0.f, 0.f, 0.f, 0.f);
  uint32_t phases = 0;  // a bit per part
  __syncthreads();  // the barriers are set up
  for (uint32_t a = i0; a < i1; a += kPos) {
    const uint32_t nk = min((uint32_t)kPos, i1 - a);
    if (a != i0) {
      __syncthreads();
      fetch(a, a + nk);
    }
    if (FUSE && a + nk == pos + 1 && warp == kWarps - 1) {  // the step's own row takes the last place
      float* dst = ks + (size_t)(nk - 1) * kw;
      key_row(p, row, 0, pos, dst, lane);
      if (head0 == 0) {
        __syncwarp();
        for (uint32_t e = lane; e < kw; e += 32) base[(size_t)pos * kw + e] = dst[e];
      }
    }
    __syncthreads();
    // ---- scores: two positions of a warp at a time, as they arrive ----
    for (uint32_t i = 0; i < (uint32_t)kParts; ++i) {
      if (i * kPart < coming) {
        if (!mbar_wait(&full[i], phases >> i & 1u)) s_abort = 1;
        phases ^= 1u << i;
      }
      const uint32_t k0 = i * kPart + 2 * warp;
      if (k0 >= nk) continue;
      const float4 *ka = reinterpret_cast<const float4*>(ks + (size_t)k0 * kw), *kb = reinterpret_cast<const float4*>(ks + (size_t)min(k0 + 1, nk - 1) * kw);
      float z[2 * kHeads];
#pragma unroll
      for (int i = 0; i < 2 * kHeads; ++i) z[i] = 0.0f;
#pragma unroll
      for (int j = 0; j < NE; ++j) {
        const uint32_t f = lane + 32 * j;
        if (f < w4) {
          const float4 va = ka[f], vb = kb[f];
#pragma unroll
          for (int h = 0; h < kHeads; ++h) { z[h] = dot4(q[h][j], va, z[h]); z[kHeads + h] = dot4(q[h][j], vb, z[kHeads + h]); }
        }
      }
      // every exchange halves what a lane holds; lane bits 0, 1, 2 end up as position and head
      uint32_t idx = 0;
#pragma unroll
      for (int s = 0; s < 5; ++s) {
        const int have = 2 * kHeads >> s;
        const uint32_t bit = 1u << s;
        if (have > 1) {
          const bool hi = lane & bit;
#pragma unroll
          for (int i = 0; i < have / 2; ++i) {
            const float send = hi ? z[i] : z[i + have / 2], keep = hi ? z[i + have / 2] : z[i];
            z[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, bit);
          }
          idx += hi ? have / 2 : 0;
        } else {
          z[0] += __shfl_xor_sync(0xFFFFFFFFu, z[0], bit);
        }
      }
      if (lane < 2 * kHeads && k0 + idx / kHeads < nk) ps[idx % kHeads][k0 + idx / kHeads] = z[0] * p.scale;
    }
    __syncthreads();
    if (warp < kHeads) {
      float* pr = ps[warp];
      const float a0 = lane < nk ? pr[lane] : -INFINITY, a1 = lane + 32 < nk ? pr[lane + 32] : -INFINITY;
      const float m_old = mr[warp], m_new = fmaxf(m_old, warp_max(fmaxf(a0, a1)));
      const float e0 = lane < nk ? expf(a0 - m_new) : 0.0f, e1 = lane + 32 < nk ? expf(a1 - m_new) : 0.0f;
      const float sum = warp_sum(e0 + e1), corr = m_old == -INFINITY ? 0.0f : expf(m_old - m_new);
      pr[lane] = e0;  // zeros past the last position
      pr[lane + 32] = e1;
      __syncwarp();
      if (lane == 0) { mr[warp] = m_new; lr[warp] = fmaf(lr[warp], corr, sum); cr[warp] = corr; }
    }
    __syncthreads();
    // ---- values ----
#pragma unroll
    for (int h = 0; h < kHeads; ++h) {
      const float corr = cr[h];
#pragma unroll
      for (int j = 0; j < NV; ++j) { acc[h][j].x *= corr; acc[h][j].y *= corr; acc[h][j].z *= corr; acc[h][j].w *= corr; }
    }
    const uint32_t ke = min(nk, (grp + 1) * per_group);
    for (uint32_t k = grp * per_group; k < ke; k += 4) {
      float4 w[kHeads];
#pragma unroll
      for (int h = 0; h < kHeads; ++h) w[h] = *reinterpret_cast<const float4*>(&ps[h][k]);
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const uint32_t f = col + vcols * j;
        if (f < v4) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float4 v = k + e < nk ? reinterpret_cast<const float4*>(ks + (size_t)(k + e) * kw)[f] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int h = 0; h < kHeads; ++h) {
              const float x = e == 0 ? w[h].x : e == 1 ? w[h].y : e == 2 ? w[h].z : w[h].w;
              acc[h][j].x = fmaf(x, v.x, acc[h][j].x); acc[h][j].y = fmaf(x, v.y, acc[h][j].y);
              acc[h][j].z = fmaf(x, v.z, acc[h][j].z); acc[h][j].w = fmaf(x, v.w, acc[h][j].w);
            }
          }
        }
      }
    }
  }
  // ---- the groups of positions come together: os [groups][kHeads][vdp] in the rows' place ----
  __syncthreads();
  if (s_abort && tid == 0 && p.status) atomicCAS(p.status, 0, 3);  // the results are void
  float4* os = reinterpret_cast<float4*>(sm);
#pragma unroll
  for (int h = 0; h < kHeads; ++h)
#pragma unroll
    for (int j = 0; j < NV; ++j)
      if (col + vcols * j < v4) os[((size_t)grp * kHeads + h) * v4 + col + vcols * j] = acc[h][j];
  __syncthreads();
  auto whole = [&](uint32_t it) {  // piece it % v4 of head it / v4
    float4 s = os[it];
    for (uint32_t g = 1; g < groups; ++g) {
      const float4 v = os[(size_t)g * kHeads * v4 + it];
      s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
    }
    return s;
  };
  const uint32_t items = nh * v4, hstride = p.vdp + 4;
  float* mine = p.scratch + (((size_t)token * H + head0) * shares + share) * hstride;  // [token][head][share][values, maximum, sum]
  for (uint32_t it = tid; it < items; it += kThreads) *reinterpret_cast<float4*>(mine + (size_t)(it / v4) * shares * hstride + 4 * (it % v4)) = whole(it);
  if (tid < nh) *reinterpret_cast<float2*>(mine + (size_t)tid * shares * hstride + p.vdp) = make_float2(mr[tid], lr[tid]);
}

// What the shares of one head left, put together: piece f of the values, by a thread; every warp of the CTA must call it
// with all of its lanes (a lane weighs a share).
__device__ __forceinline__ float share_weight(const float* all, uint32_t shares, uint32_t vdp, uint32_t lane) {
  const float2 ml = lane < shares ? __ldcg(reinterpret_cast<const float2*>(all + (size_t)lane * (vdp + 4) + vdp)) : make_float2(-INFINITY, 0.0f);
  const float M = warp_max(ml.x), w = ml.x == -INFINITY ? 0.0f : expf(ml.x - M);
  return w / warp_sum(ml.y * w);
}
__device__ __forceinline__ float4 merged_piece(const float* all, uint32_t shares, uint32_t vdp, uint32_t f, bool in, uint32_t lane) {
  constexpr uint32_t kBatch = 16;  // shares requested together, the first ones before their weights are known
  float4 v[kBatch], o = make_float4(0.f, 0.f, 0.f, 0.f);
  float w = 0.0f;
  for (uint32_t s0 = 0; s0 < shares; s0 += kBatch) {
#pragma unroll
    for (uint32_t s = 0; s < kBatch; ++s)
      v[s] = in && s0 + s < shares ? __ldcg(reinterpret_cast<const float4*>(all + (size_t)(s0 + s) * (vdp + 4)) + f) : make_float4(0.f, 0.f, 0.f, 0.f);
    if (s0 == 0) w = share_weight(all, shares, vdp, lane);
#pragma unroll
    for (uint32_t s = 0; s < kBatch; ++s) {
      const float x = __shfl_sync(0xFFFFFFFFu, w, (s0 + s) & 31u);  // zero past the last share
      o.x = fmaf(x, v[s].x, o.x); o.y = fmaf(x, v[s].y, o.y); o.z = fmaf(x, v[s].z, o.z); o.w = fmaf(x, v[s].w, o.w);
    }
  }
  return o;
}

// grid (heads, tokens): the merged result itself, times the gate
__global__ void __launch_bounds__(128) latent_merge_kernel(const SpanParams p, uint32_t shares) {
  const uint32_t head = blockIdx.x, token = blockIdx.y, lane = threadIdx.x & 31, v4 = p.vdp / 4;
  grid_dependency_wait();
  grid_launch_dependents();
  if ((uint32_t)*p.len + token % p.T >= p.cap) return;
  const float* all = p.scratch + ((size_t)token * p.rep + head) * shares * (p.vdp + 4);
  const float g = p.gate ? p.gate[(size_t)token * p.ld_gate + head] : 1.0f;
  for (uint32_t f0 = 0; f0 < v4; f0 += 128) {
    const uint32_t f = f0 + threadIdx.x;
    const float4 v = merged_piece(all, shares, p.vdp, f, f < v4, lane);
    if (f >= v4) continue;
    const float y[4] = {v.x * g, v.y * g, v.z * g, v.w * g};
    const size_t o = (size_t)token * p.out_ld + (size_t)head * (p.out_step ? p.out_step : p.vd) + 4 * f;
#pragma unroll
    for (uint32_t e = 0; e < 4; ++e)
      if (4 * f + e < p.vd) store_from_f32(p.out, p.out_dtype, o + e, y[e]);
  }
}

// grid (blocks of kORows rows, heads, tokens): the merged result through the head's part of a projection, rows of w [vd] at
// head * block_n; a warp owns four rows, whose weights are requested ahead of the dependency wait
constexpr uint32_t kORows = 32;
template <typename WT>
__global__ void __launch_bounds__(256) latent_project_kernel(const SpanParams p, uint32_t shares, const WT* w, uint32_t ldw, uint32_t block_n, uint32_t rows, void* out,
                                                             uint32_t out_ld, int out_dtype) {
  extern __shared__ __align__(16) float xs[];  // [vdp]
  const uint32_t head = blockIdx.y, token = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, v4 = p.vdp / 4;
  const uint32_t r0 = blockIdx.x * kORows + 4 * warp;
  const WT* wr = w + ((size_t)head * block_n + r0) * ldw;
  constexpr int kHold = 4;  // pieces of four elements per row and lane, held in registers: 512 elements
  auto piece = [&](uint32_t r, uint32_t f) {  // rows of w are ldw >= vd apart, ldw a multiple of 8, zero past vd
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (r0 + r < rows && 4 * f < ldw && f < v4) {
      if constexpr (sizeof(WT) == 4) x = *reinterpret_cast<const float4*>(wr + (size_t)r * ldw + 4 * f);
      else {
        const uint2 u = *reinterpret_cast<const uint2*>(wr + (size_t)r * ldw + 4 * f);
        x = make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xFFFF0000u));
      }
    }
    return x;
  };
  float4 hold[4][kHold];
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int j = 0; j < kHold; ++j) hold[r][j] = piece(r, lane + 32 * j);
  grid_dependency_wait();
  grid_launch_dependents();
  const bool over = (uint32_t)*p.len + token % p.T >= p.cap;
  const float* all = p.scratch + ((size_t)token * p.rep + head) * shares * (p.vdp + 4);
  const float g = p.gate ? p.gate[(size_t)token * p.ld_gate + head] : 1.0f;
  if (!over)
    for (uint32_t f0 = 0; f0 < v4; f0 += 256) {
      if (f0 + 32 * warp >= v4) break;  // whole warps
      const uint32_t f = f0 + tid;
      const float4 v = merged_piece(all, shares, p.vdp, f, f < v4, lane);
      if (f < v4) reinterpret_cast<float4*>(xs)[f] = make_float4(v.x * g, v.y * g, v.z * g, v.w * g);
    }
  __syncthreads();
  if (over) return;
  float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
  for (int j = 0; j < kHold; ++j) {
    const uint32_t f = lane + 32 * j;
    const float4 x = f < v4 ? reinterpret_cast<const float4*>(xs)[f] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < 4; ++r) acc[r] = dot4(hold[r][j], x, acc[r]);
  }
  for (uint32_t f = lane + 32 * kHold; f < v4; f += 32) {
    const float4 x = reinterpret_cast<const float4*>(xs)[f];
#pragma unroll
    for (int r = 0; r < 4; ++r) acc[r] = dot4(piece(r, f), x, acc[r]);
  }
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const float s = warp_sum(acc[r]);
    if (lane == 0 && r0 + r < rows) store_from_f32(out, out_dtype, (size_t)token * out_ld + (size_t)head * rows + r0 + r, s);
  }
}

uint32_t latent_subs(const SpanParams& p) { return (p.rep + kHeads - 1) / kHeads; }
uint32_t latent_shares(const SpanParams& p, uint32_t B) {
  const uint64_t ctas = (uint64_t)B * latent_subs(p) * p.T;
  const uint32_t room = ctas >= 592 ? 1 : (uint32_t)(592 / ctas);
  return std::max(1u, std::min(std::min((p.cap + kPos - 1) / kPos, room), kShares));
}
size_t latent_smem(const SpanParams& p) {
  const uint32_t v4 = p.vdp / 4, vcols = v4 > 64 ? 128u : v4 > 32 ? 64u : 32u;
  return std::max((size_t)kPos * (p.kdp + p.rotp), (size_t)(kThreads / vcols) * kHeads * p.vdp) * sizeof(float);
}
template <bool FUSE, int NE, int NV>
cudaError_t latent_launch(ruai_ctx* c, const SpanParams& p, uint32_t B) {
  static bool attr_done[64] = {};
  if (!attr_done[c->ordinal & 63]) {
    cudaError_t e = cudaFuncSetAttribute(latent_attention_kernel<FUSE, NE, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return e;
    attr_done[c->ordinal & 63] = true;
  }
  const dim3 grid(B * latent_subs(p), p.T, latent_shares(p, B));
  return ruai_launch(c, latent_attention_kernel<FUSE, NE, NV>, grid, dim3(kThreads), latent_smem(p), true, p, latent_subs(p));
}
template <bool FUSE>
cudaError_t latent_dispatch(ruai_ctx* c, const SpanParams& p, uint32_t B) {
  const uint32_t w4 = (p.kdp + p.rotp) / 4, v4 = p.vdp / 4;
  if (w4 <= 64) return latent_launch<FUSE, 2, 1>(c, p, B);
  if (w4 <= 96) return latent_launch<FUSE, 3, 1>(c, p, B);
  return v4 <= 128 ? latent_launch<FUSE, 5, 1>(c, p, B) : latent_launch<FUSE, 5, 2>(c, p, B);
}

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

namespace {
template <typename WT>
cudaError_t project(ruai_ctx* c, const SpanParams& p, uint32_t B, const LatentProjection& o) {
  const uint32_t rows = o.rows;
  return ruai_launch(c, latent_project_kernel<WT>, dim3((rows + kORows - 1) / kORows, p.rep, B * p.T), dim3(256), p.vdp * sizeof(float), true, p, latent_shares(p, B),
                     (const WT*)o.w->data, o.w->ld, o.block_n, rows, o.out, o.out_ld, o.out_dtype);
}
}  // namespace

bool ruai_attn_latent_takes(const SpanParams& p) {
  return p.shared && p.maps == 1 && p.G == 1 && p.window == 0xFFFFFFFFu && p.kdp == p.vdp && p.kdp + p.rotp <= 640 && !p.q_norm && p.kd % 4 == 0 && p.q_step % 4 == 0 &&
         p.q_rot % 4 == 0 && p.ld % 4 == 0 && p.out_scale == 1.0f;
}

size_t ruai_attn_latent_scratch(const SpanParams& p, uint32_t B) {
  return (size_t)B * p.T * p.rep * latent_shares(p, B) * (p.vdp + 4) * sizeof(float);
}

int ruai_attn_latent(ruai_ctx* c, const SpanParams& p, uint32_t B, const LatentProjection* o) {
  if (p.T > 65535 || (uint64_t)B * p.T > 65535) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "a step of %u tokens is too large for this head shape", B * p.T);
  RUAI_CUDA(c, p.T == 1 ? latent_dispatch<true>(c, p, B) : latent_dispatch<false>(c, p, B));
  if (o) RUAI_CUDA(c, o->w->bits == 16 ? project<__nv_bfloat16>(c, p, B, *o) : project<float>(c, p, B, *o));
  else RUAI_CUDA(c, ruai_launch(c, latent_merge_kernel, dim3(p.rep, B * p.T), dim3(128), 0, true, p, latent_shares(p, B)));
  return RUAI_OK;
}

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
