// Latent attention of few queries, rotation tables and latent rows (see attn_latent.cuh).
//
// latent_attention_kernel: a CTA owns four heads of one query position and a share of the cached positions, which come into
// shared memory 64 at a time and serve as keys and as values.  Scores: a warp per position, its lanes across the row, the
// four queries in registers, so that a row is read once; sums of values: a thread per four elements of the row and a group of
// the positions, all four heads in registers.  The last CTA of a query merges the shares.  In the single-token step the
// kernel also rotates the queries, norms and rotates the new position's row and appends it; cached rows are requested
// ahead of the dependency wait.  Everything is f32.
#include "attn_rows.cuh"

#include <algorithm>
#include <cmath>

#include "attn_latent.cuh"

namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32, kHeads = 4, kPos = 64;
constexpr uint32_t kShares = 32;  // at most: a lane per share when they are merged

__device__ __forceinline__ float dot4(float4 a, float4 b, float s) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, s)))); }

// grid (sequences x groups of kHeads heads, T, shares); NE: four-element pieces of a row per lane, NV: of a value per thread
template <bool FUSE, int NE, int NV>
__global__ void __launch_bounds__(kThreads) latent_attention_kernel(const SpanParams p, uint32_t subs) {
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(16) float ps[kHeads][kPos];
  __shared__ float mr[kHeads], lr[kHeads], cr[kHeads], wts[kHeads][kShares];
  __shared__ unsigned s_last;
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
  auto fetch = [&](uint32_t a, uint32_t e) {  // rows that are in the cache already
    const uint32_t end = FUSE ? min(e, pos) : e;
    for (uint32_t i = a + warp; i < end; i += kWarps)
      for (uint32_t c = lane; c < w4; c += 32) cp_async16(ks + (size_t)(i - a) * kw + 4 * c, base + (size_t)i * kw + 4 * c);
  };
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
  if (over) {
    if (tid == 0 && p.status) atomicCAS(p.status, 0, 5);
    cp_async_wait();
  }
  const size_t token = (size_t)b * p.T + t;
  const float* row = p.qkv + token * p.ld;
  // ---- this lane's pieces of the queries ----
  float4 q[kHeads][NE];
#pragma unroll
  for (int h = 0; h < kHeads; ++h) {
#pragma unroll
    for (int j = 0; j < NE; ++j) {
      const uint32_t f = lane + 32 * j;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if ((uint32_t)h < nh && f < w4 && !over) {
        if (!FUSE) {
          v = *reinterpret_cast<const float4*>(p.q + (token * H + head0 + h) * kw + 4 * f);
        } else if (4 * f < p.kdp) {
          const float* src = p.q_main + (token * H + head0 + h) * p.kd + 4 * f;
          if (p.kd % 4 == 0) v = *reinterpret_cast<const float4*>(src);
          else {
            v.x = src[0];
            v.y = 4 * f + 1 < p.kd ? src[1] : 0.f; v.z = 4 * f + 2 < p.kd ? src[2] : 0.f; v.w = 4 * f + 3 < p.kd ? src[3] : 0.f;
          }
        } else {  // two pairs; past the rotated ones the projection holds zeros
          const uint32_t e = 4 * f - p.kdp, i = e / 2, pairs = p.rot / 2;
          const float2* cs = p.table + (size_t)pos * pairs;
          const float4 u = *reinterpret_cast<const float4*>(row + (size_t)(head0 + h) * p.q_step + p.q_rot + e);
          const float2 c0 = i < pairs ? cs[i] : make_float2(1.f, 0.f), c1 = i + 1 < pairs ? cs[i + 1] : make_float2(1.f, 0.f);
          v.x = fmaf(u.x, c0.x, -(u.y * c0.y)); v.y = fmaf(u.y, c0.x, u.x * c0.y);
          v.z = fmaf(u.z, c1.x, -(u.w * c1.y)); v.w = fmaf(u.w, c1.x, u.z * c1.y);
        }
      }
      q[h][j] = v;
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
    cp_async_wait();
    __syncthreads();
    // ---- scores: two positions of a warp at a time ----
    for (uint32_t k0 = 2 * warp; k0 < nk; k0 += 2 * kWarps) {
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
  const uint32_t items = nh * v4;
  auto finish = [&](uint32_t it, float4 v) {
    const uint32_t head = head0 + it / v4;
    const float g = p.gate ? p.gate[token * p.ld_gate + head] : 1.0f;
    const float y[4] = {v.x * g, v.y * g, v.z * g, v.w * g};
    const size_t o = token * p.out_ld + (size_t)head * (p.out_step ? p.out_step : p.vd) + 4 * (it % v4);
#pragma unroll
    for (uint32_t e = 0; e < 4; ++e)
      if (4 * (it % v4) + e < p.vd) store_from_f32(p.out, p.out_dtype, o + e, y[e]);
  };
  if (shares == 1) {
    if (over) return;
    for (uint32_t it = tid; it < items; it += kThreads) {
      const float inv = 1.0f / lr[it / v4];
      float4 v = whole(it);
      v.x *= inv; v.y *= inv; v.z *= inv; v.w *= inv;
      finish(it, v);
    }
    return;
  }
  const size_t query = (size_t)blockIdx.x * p.T + t, hstride = p.vdp + 4, stride = kHeads * hstride;
  float* mine = p.scratch + (query * shares + share) * stride;
  for (uint32_t it = tid; it < items; it += kThreads) *reinterpret_cast<float4*>(mine + (it / v4) * hstride + 4 * (it % v4)) = whole(it);
  if (tid < nh) { mine[tid * hstride + p.vdp] = mr[tid]; mine[tid * hstride + p.vdp + 1] = lr[tid]; }
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    s_last = atomicAdd(p.counters + query, 1u) == shares - 1 ? 1u : 0u;
    if (s_last) p.counters[query] = 0;
  }
  __syncthreads();
  if (!s_last || over) return;
  __threadfence();
  const float* all = p.scratch + query * shares * stride;
  if (warp < nh) {  // weights of the shares, a lane per share
    const float* src = all + lane * stride + warp * hstride + p.vdp;
    const float m = lane < shares ? __ldcg(src) : -INFINITY, l = lane < shares ? __ldcg(src + 1) : 0.0f;
    const float M = warp_max(m), w = m == -INFINITY ? 0.0f : expf(m - M), L = warp_sum(l * w);
    wts[warp][lane] = w / L;
  }
  __syncthreads();
  for (uint32_t it = tid; it < items; it += kThreads) {
    const float* src = all + (it / v4) * hstride + 4 * (it % v4);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    constexpr uint32_t kBatch = 8;  // shares requested together
    for (uint32_t s0 = 0; s0 < shares; s0 += kBatch) {
      float4 v[kBatch];
#pragma unroll
      for (uint32_t s = 0; s < kBatch; ++s) v[s] = s0 + s < shares ? __ldcg(reinterpret_cast<const float4*>(src + (s0 + s) * stride)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (uint32_t s = 0; s < kBatch; ++s) {
        const float w = s0 + s < shares ? wts[it / v4][s0 + s] : 0.0f;
        o.x = fmaf(w, v[s].x, o.x); o.y = fmaf(w, v[s].y, o.y); o.z = fmaf(w, v[s].z, o.z); o.w = fmaf(w, v[s].w, o.w);
      }
    }
    finish(it, o);
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

bool ruai_attn_latent_takes(const SpanParams& p) {
  return p.shared && p.maps == 1 && p.G == 1 && p.window == 0xFFFFFFFFu && p.kdp == p.vdp && p.kdp + p.rotp <= 640 && !p.q_norm && p.q_step % 4 == 0 &&
         p.q_rot % 4 == 0 && p.ld % 4 == 0 && p.out_scale == 1.0f;
}

size_t ruai_attn_latent_scratch(const SpanParams& p, uint32_t B, size_t* counters) {
  const uint32_t shares = latent_shares(p, B);
  *counters = 0;
  if (shares == 1) return 0;
  *counters = (size_t)B * latent_subs(p) * p.T;
  return *counters * shares * kHeads * (p.vdp + 4) * sizeof(float);
}

int ruai_attn_latent(ruai_ctx* c, const SpanParams& p, uint32_t B) {
  if (p.T > 65535) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "a step of %u tokens is too large for this head shape", p.T);
  RUAI_CUDA(c, p.T == 1 ? latent_dispatch<true>(c, p, B) : latent_dispatch<false>(c, p, B));
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
