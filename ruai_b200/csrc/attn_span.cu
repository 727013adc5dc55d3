// Attention of few query positions over a span of the cache (see attn_span.cuh): a position sees itself, the window
// behind it and the kept first positions.
//
// A CTA owns (sequence, key / value head, some of its query heads), one query position and a share of the visible
// positions, which are numbered without the gap between the kept ones and the window, so that the shares are even and
// nothing invisible is read.  Rows of scores are (map, head).  Positions come into shared memory some at a time (keys
// padded so that a thread per key reads them without bank conflicts); scores by thread = (key, row), running softmax by
// warp = row, values by thread = (row, four elements).  The last CTA of a query to finish merges the shares, combines
// the maps and applies the output norm.  In the single-token step the kernel also norms the query and the new key and
// appends the new position; cached positions are fetched ahead of the dependency wait.
//
// SHARED: latent attention in its absorbed form, for rows that attn_latent.cu does not take.  All heads share one row per
// position, whose front is also the value; a thread takes its key through several rows of scores at a time, and a value
// through several rows of sums.
//
// Everything is f32.
#include "attn_rows.cuh"

#include <algorithm>

#include "decode_ops.cuh"

namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32, kItems = 4;

// Norms the queries into p.q and appends keys and values: one warp per row of (token; query head and map, key head and
// map, value head).
__global__ void __launch_bounds__(kThreads) span_append_kernel(const SpanParams p, uint32_t rows) {
  grid_dependency_wait();
  grid_launch_dependents();
  const uint32_t lane = threadIdx.x & 31, nq = p.G * p.rep * p.maps, nk = p.G * p.maps, per = nq + nk + (p.shared ? 0 : p.G);
  const uint32_t i = blockIdx.x * kWarps + (threadIdx.x >> 5);
  if (i >= rows * per) return;
  const uint32_t row = i / per, e = i % per, b = row / p.T, pos = (uint32_t)*p.len + row % p.T;
  const float* src = p.qkv + (size_t)row * p.ld;
  if (pos >= p.cap) {
    if (lane == 0 && p.status) atomicCAS(p.status, 0, 5);
    return;
  }
  if (e < nq) {
    query_row(p, row, src, e, nq, pos, p.q + ((size_t)row * nq + e) * ((p.qd ? p.qdp : p.kdp) + p.rotp), lane);
  } else if (e < nq + nk) {
    const uint32_t g = (e - nq) / p.maps, mp = (e - nq) % p.maps;
    key_row(p, src, e - nq, pos, p.kcache + (((size_t)b * p.G + g) * p.cap + pos) * (p.maps * p.kdp + p.rotp) + mp * p.kdp, lane);
  } else {
    const uint32_t g = e - nq - nk;
    norm_row(src + p.v_off + (size_t)g * p.vd, nullptr, 0.0f, p.vd, p.vdp, p.vcache + (((size_t)b * p.G + g) * p.cap + pos) * p.vdp, lane);
  }
}

struct Plan {  // how a launch shares the work out
  uint32_t rc, subs, kc, splits;  // query heads per CTA, CTAs per key / value head, positions per chunk
};

// grid (B * G * subs, T, splits)
template <bool FUSE, bool SHARED>
__global__ void __launch_bounds__(kThreads) span_attention_kernel(const SpanParams p, const Plan pl) {
  extern __shared__ __align__(16) float sm[];
  __shared__ unsigned s_last;
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t bg = blockIdx.x / pl.subs, sub = blockIdx.x % pl.subs, b = bg / p.G, g = bg % p.G, t = blockIdx.y, split = blockIdx.z;
  const uint32_t kw = p.maps * p.kdp + p.rotp, qw = p.kdp + p.rotp, kst = kw + 4, k4 = qw / 4, v4 = p.vdp / 4, R = pl.rc * p.maps, kc = pl.kc;
  const uint32_t own_v = SHARED ? 0 : p.vdp, vst4 = SHARED ? kst / 4 : v4;  // float4s between the values of two positions
  float* ks = sm;                                      // [kc][kw + 4]
  float* vs = SHARED ? ks : ks + (size_t)kc * kst;     // [kc][vdp]
  float* qs = ks + (size_t)kc * (kst + own_v);         // [R][qw]
  float* knew = qs + (size_t)R * qw;                   // [kw]
  float* vnew = knew + kw;                             // [vdp]
  float* ps = vnew + own_v;                            // [R][kc]
  float* mr = ps + (size_t)R * kc;       // [R] running maximum
  float* lr = mr + R;                    // [R] running sum
  float* cr = lr + R;                    // [R] factor of the sums so far
  float* kbase = p.kcache + (size_t)bg * p.cap * kw;
  float* vbase = p.vcache + (size_t)bg * p.cap * p.vdp;
  uint32_t pos = 0, lo = 0, sink = 0, n = 0, i0 = 0, i1 = 0;
  bool over = false;
  auto plan = [&]() {
    pos = (uint32_t)__ldcg(p.len) + t;
    over = pos >= p.cap;  // the host grows the cache ahead of the step: touch nothing beyond it, tell the host
    lo = pos + 1 > p.window ? pos + 1 - p.window : 0;
    sink = min(p.keep, lo);
    n = sink + (pos - lo) + 1;
    const uint32_t per = (n + pl.splits - 1) / pl.splits;
    i0 = over ? 0 : min(n, split * per);
    i1 = over ? 0 : min(n, i0 + per);
  };
  auto place = [&](uint32_t i) { return i < sink ? i : lo + i - sink; };
  // positions [a, e) of the list into shared memory; the fused step's own position (the last of the list) is left out
  auto fetch = [&](uint32_t a, uint32_t e) {
    const uint32_t cnt = e - a, kq = kw / 4, unit = kq + own_v / 4, cached = FUSE ? n - 1 : n;
    for (uint32_t i = warp; i < cnt; i += kWarps) {  // a warp per position
      if (a + i >= cached) break;
      const uint32_t at = place(a + i);
      const float *kp = kbase + (size_t)at * kw, *vp = vbase + (size_t)at * p.vdp;
      for (uint32_t c = lane; c < unit; c += 32) {
        if (c < kq) cp_async16(ks + (size_t)i * kst + 4 * c, kp + 4 * c);
        else cp_async16(vs + (size_t)i * p.vdp + 4 * (c - kq), vp + 4 * (c - kq));
      }
    }
  };
  if (FUSE) {  // cached positions and the position word are earlier steps' work
    plan();
    fetch(i0, min(i1, i0 + kc));
  }
  grid_dependency_wait();
  grid_launch_dependents();
  if (!FUSE) {
    plan();
    fetch(i0, min(i1, i0 + kc));
  }
  if (over && tid == 0 && p.status) atomicCAS(p.status, 0, 5);
  const bool owner = FUSE && i1 == n && i1 > i0;
  const uint32_t head0 = g * p.rep + sub * pl.rc;
  const float* row = p.qkv + (size_t)(b * p.T + t) * p.ld;
  for (uint32_t i = warp; i < R + (owner && !over ? p.maps + (SHARED ? 0 : 1) : 0); i += kWarps) {
    if (i < R) {
      const uint32_t mp = i / pl.rc, hh = i % pl.rc, e = (head0 + hh) * p.maps + mp, nq = p.G * p.rep * p.maps;
      if (FUSE) { if (!over) query_row(p, b, row, e, nq, pos, qs + (size_t)i * qw, lane); }
      else norm_row(p.q + ((size_t)(b * p.T + t) * nq + e) * qw, nullptr, 0.0f, qw, qw, qs + (size_t)i * qw, lane);
    } else if (i < R + p.maps) {
      const uint32_t mp = i - R;
      key_row(p, row, g * p.maps + mp, pos, knew + mp * p.kdp, lane);
    } else {
      norm_row(row + p.v_off + (size_t)g * p.vd, nullptr, 0.0f, p.vd, p.vdp, vnew, lane);
    }
  }
  for (uint32_t i = tid; i < R; i += kThreads) {  // the sink is a first term without a value, in one of the shares
    const bool sink_here = p.sink && split == 0;
    mr[i] = sink_here ? p.sink[head0 + i] : -INFINITY;
    lr[i] = sink_here ? 1.0f : 0.0f;
  }
  __syncthreads();
  if (owner && sub == 0) {
    for (uint32_t e = tid; e < kw; e += kThreads) kbase[(size_t)pos * kw + e] = knew[e];
    if (!SHARED)
      for (uint32_t e = tid; e < p.vdp; e += kThreads) vbase[(size_t)pos * p.vdp + e] = vnew[e];
  }
  const uint32_t items = R * v4;
  float4 acc[kItems];
#pragma unroll
  for (int u = 0; u < kItems; ++u) acc[u] = make_float4(0.f, 0.f, 0.f, 0.f);
  const uint32_t key = tid % kc, rg = tid / kc, rgs = kThreads / kc;
  for (uint32_t a = i0; a < i1; a += kc) {
    const uint32_t nk = min(kc, i1 - a);
    if (a != i0) {
      __syncthreads();
      fetch(a, a + nk);
    }
    if (owner && a + nk == n) {  // the step's own position takes the last place
      for (uint32_t e = tid; e < kw; e += kThreads) ks[(size_t)(nk - 1) * kst + e] = knew[e];
      if (!SHARED)
        for (uint32_t e = tid; e < p.vdp; e += kThreads) vs[(size_t)(nk - 1) * p.vdp + e] = vnew[e];
    }
    cp_async_wait();
    __syncthreads();
    if (SHARED) {
      constexpr int kR = 4;
      if (key < nk) {
        const float4* kp = reinterpret_cast<const float4*>(ks + (size_t)key * kst);
        for (uint32_t r0 = rg; r0 < R; r0 += kR * rgs) {
          const float4* qp[kR];
          float s0[kR], s1[kR];
#pragma unroll
          for (int u = 0; u < kR; ++u) {
            qp[u] = reinterpret_cast<const float4*>(qs + (size_t)min(r0 + u * rgs, R - 1) * qw);
            s0[u] = 0.0f; s1[u] = 0.0f;
          }
#pragma unroll 2
          for (uint32_t e = 0; e < k4; ++e) {
            const float4 kv = kp[e];
#pragma unroll
            for (int u = 0; u < kR; ++u) {
              if (r0 + u * rgs < R) {
                const float4 qv = qp[u][e];
                s0[u] = fmaf(qv.x, kv.x, s0[u]); s1[u] = fmaf(qv.y, kv.y, s1[u]); s0[u] = fmaf(qv.z, kv.z, s0[u]); s1[u] = fmaf(qv.w, kv.w, s1[u]);
              }
            }
          }
#pragma unroll
          for (int u = 0; u < kR; ++u)
            if (r0 + u * rgs < R) ps[(size_t)(r0 + u * rgs) * kc + key] = (s0[u] + s1[u]) * p.scale;
        }
      }
    } else if (key < nk) {
      for (uint32_t r = rg; r < R; r += rgs) {
        const float4* kp = reinterpret_cast<const float4*>(ks + (size_t)key * kst + (r / pl.rc) * p.kdp);
        const float4* qp = reinterpret_cast<const float4*>(qs + (size_t)r * p.kdp);
        float s0 = 0.0f, s1 = 0.0f;
#pragma unroll 4
        for (uint32_t e = 0; e < k4; ++e) {
          const float4 kv = kp[e], qv = qp[e];
          s0 = fmaf(qv.x, kv.x, s0); s1 = fmaf(qv.y, kv.y, s1); s0 = fmaf(qv.z, kv.z, s0); s1 = fmaf(qv.w, kv.w, s1);
        }
        ps[(size_t)r * kc + key] = (s0 + s1) * p.scale;
      }
    }
    __syncthreads();
    for (uint32_t r = warp; r < R; r += kWarps) {
      float* pr = ps + (size_t)r * kc;
      const float a0 = lane < nk ? pr[lane] : -INFINITY, a1 = lane + 32 < nk ? pr[lane + 32] : -INFINITY;  // kc <= 64
      const float m_old = mr[r], m_new = fmaxf(m_old, warp_max(fmaxf(a0, a1)));
      const float e0 = lane < nk ? expf(a0 - m_new) : 0.0f, e1 = lane + 32 < nk ? expf(a1 - m_new) : 0.0f;
      const float sum = warp_sum(e0 + e1), corr = m_old == -INFINITY ? 0.0f : expf(m_old - m_new);
      if (lane < nk) pr[lane] = e0;
      if (lane + 32 < nk) pr[lane + 32] = e1;
      __syncwarp();
      if (lane == 0) { mr[r] = m_new; lr[r] = fmaf(lr[r], corr, sum); cr[r] = corr; }
    }
    __syncthreads();
    if (SHARED && kThreads % v4 == 0) {  // a thread's items are one place of several rows
      const uint32_t r0 = tid / v4, dr = kThreads / v4;
      const float4* vp = reinterpret_cast<const float4*>(vs) + tid % v4;
#pragma unroll
      for (int u = 0; u < kItems; ++u) {
        const float corr = cr[min(r0 + u * dr, R - 1)];
        acc[u].x *= corr; acc[u].y *= corr; acc[u].z *= corr; acc[u].w *= corr;
      }
#pragma unroll 4
      for (uint32_t q = 0; q < nk; ++q) {
        const float4 v = vp[(size_t)q * vst4];
#pragma unroll
        for (int u = 0; u < kItems; ++u) {
          if (r0 + u * dr < R) {
            const float w = ps[(size_t)(r0 + u * dr) * kc + q];
            acc[u].x = fmaf(w, v.x, acc[u].x); acc[u].y = fmaf(w, v.y, acc[u].y); acc[u].z = fmaf(w, v.z, acc[u].z); acc[u].w = fmaf(w, v.w, acc[u].w);
          }
        }
      }
      continue;
    }
#pragma unroll
    for (int u = 0; u < kItems; ++u) {
      const uint32_t it = tid + u * kThreads;
      if (it < items) {
        const uint32_t r = it / v4, c = it % v4;
        const float corr = cr[r];
        const float* pr = ps + (size_t)r * kc;
        const float4* vp = reinterpret_cast<const float4*>(vs) + c;
        float4 o = make_float4(acc[u].x * corr, acc[u].y * corr, acc[u].z * corr, acc[u].w * corr);
#pragma unroll 4
        for (uint32_t q = 0; q < nk; ++q) {
          const float w = pr[q];
          const float4 v = vp[(size_t)q * vst4];
          o.x = fmaf(w, v.x, o.x); o.y = fmaf(w, v.y, o.y); o.z = fmaf(w, v.z, o.z); o.w = fmaf(w, v.w, o.w);
        }
        acc[u] = o;
      }
    }
  }
  __syncthreads();
  // ---- the shares come together; the merged sums divided by their totals land in os [R][vdp] ----
  float* os = sm;  // keys, values and queries are no longer needed
  if (pl.splits == 1) {
#pragma unroll
    for (int u = 0; u < kItems; ++u) {
      const uint32_t it = tid + u * kThreads;
      if (it < items) {
        const float inv = 1.0f / lr[it / v4];
        reinterpret_cast<float4*>(os)[it] = make_float4(acc[u].x * inv, acc[u].y * inv, acc[u].z * inv, acc[u].w * inv);
      }
    }
  } else {
    const size_t query = (size_t)blockIdx.x * p.T + t, stride = (size_t)R * (p.vdp + 4);
    float* mine = p.scratch + (query * pl.splits + split) * stride;
#pragma unroll
    for (int u = 0; u < kItems; ++u) {
      const uint32_t it = tid + u * kThreads;
      if (it < items) *reinterpret_cast<float4*>(mine + (size_t)(it / v4) * (p.vdp + 4) + 4 * (it % v4)) = acc[u];
    }
    for (uint32_t r = tid; r < R; r += kThreads) { mine[(size_t)r * (p.vdp + 4) + p.vdp] = mr[r]; mine[(size_t)r * (p.vdp + 4) + p.vdp + 1] = lr[r]; }
    __threadfence();
    __syncthreads();
    if (tid == 0) {
      s_last = atomicAdd(p.counters + query, 1u) == pl.splits - 1 ? 1u : 0u;
      if (s_last) p.counters[query] = 0;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    const float* all = p.scratch + query * pl.splits * stride;
    for (uint32_t r = warp; r < R; r += kWarps) {  // weights of the shares, a lane per share (at most 32)
      const float* src = all + lane * stride + (size_t)r * (p.vdp + 4) + p.vdp;
      const float m = lane < pl.splits ? __ldcg(src) : -INFINITY, l = lane < pl.splits ? __ldcg(src + 1) : 0.0f;
      const float M = warp_max(m), w = m == -INFINITY ? 0.0f : expf(m - M), L = warp_sum(l * w);
      ps[r * 32 + lane] = w / L;  // kc >= 32, or R * 32 floats reserved
    }
    __syncthreads();
#pragma unroll
    for (int u = 0; u < kItems; ++u) {
      const uint32_t it = tid + u * kThreads;
      if (it < items) {
        const uint32_t r = it / v4, c = it % v4;
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        constexpr uint32_t kBatch = 16;  // shares requested together
        for (uint32_t s0 = 0; s0 < pl.splits; s0 += kBatch) {
          float4 v[kBatch];
#pragma unroll
          for (uint32_t s = 0; s < kBatch; ++s)
            v[s] = s0 + s < pl.splits ? __ldcg(reinterpret_cast<const float4*>(all + (s0 + s) * stride + (size_t)r * (p.vdp + 4) + 4 * c)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (uint32_t s = 0; s < kBatch; ++s) {
            const float w = s0 + s < pl.splits ? ps[r * 32 + s0 + s] : 0.0f;
            o.x = fmaf(w, v[s].x, o.x); o.y = fmaf(w, v[s].y, o.y); o.z = fmaf(w, v[s].z, o.z); o.w = fmaf(w, v[s].w, o.w);
          }
        }
        acc[u] = o;
      }
    }
#pragma unroll
    for (int u = 0; u < kItems; ++u) {
      const uint32_t it = tid + u * kThreads;
      if (it < items) reinterpret_cast<float4*>(os)[it] = acc[u];
    }
  }
  __syncthreads();
  if (over) return;
  // ---- combine the maps, a warp per head ----
  const float lam = p.maps == 2 ? *p.lambda : 0.0f;
  for (uint32_t hh = warp; hh < pl.rc; hh += kWarps) {
    const float *a1 = os + (size_t)hh * p.vdp, *a2 = os + (size_t)(pl.rc + hh) * p.vdp;
    const size_t o = (size_t)(b * p.T + t) * p.out_ld + (size_t)(head0 + hh) * (p.out_step ? p.out_step : p.vd);
    float f = p.out_scale;
    if (p.gate) f *= p.gate[(size_t)(b * p.T + t) * p.ld_gate + head0 + hh];
    if (p.maps == 2) {
      float ss = 0.0f;
      for (uint32_t e = lane; e < p.vd; e += 32) { const float d = a1[e] - lam * a2[e]; ss = fmaf(d, d, ss); }
      ss = warp_sum(ss);
      f *= 1.0f / sqrtf(ss / (float)p.vd + p.eps);
    }
    for (uint32_t e = lane; e < p.vd; e += 32) store_from_f32(p.out, p.out_dtype, o + e, (p.maps == 2 ? a1[e] - lam * a2[e] : a1[e]) * f);
  }
}

size_t plan_smem(const SpanParams& p, const Plan& pl) {
  const size_t R = (size_t)pl.rc * p.maps, kw = (size_t)p.maps * p.kdp + p.rotp, own_v = p.shared ? 0 : p.vdp;
  const size_t floats = (size_t)pl.kc * (kw + 4 + own_v) + R * (p.kdp + p.rotp) + kw + own_v + R * (pl.kc > 32 ? pl.kc : 32) + 3 * R;
  const size_t outs = R * p.vdp;  // reuses the front
  return (floats > outs + R * 64 ? floats : outs + R * 64) * sizeof(float);
}

// As many query heads of a group per CTA as still leave CTAs for most of the SMs (fewer heads: the group's keys are read
// again from the L2, but the shares are fewer and the last CTA of a query has less to merge), one chunk of positions per
// CTA unless the grid is large without that.
bool make_plan(const SpanParams& p, uint32_t B, Plan* pl) {
  const uint64_t span = (uint64_t)p.keep + p.window;
  const uint32_t most = span < p.cap ? (uint32_t)span : p.cap;
  bool found = false;
  for (uint32_t rc = p.rep; rc >= 1; --rc) {
    if (p.rep % rc) continue;
    const uint32_t R = rc * p.maps;
    if ((rc > 1 && R > 16) || (size_t)R * p.vdp / 4 > (size_t)kThreads * kItems) continue;
    for (uint32_t kc : {64u, 32u, 16u}) {
      Plan q;
      q.rc = rc; q.subs = p.rep / rc; q.kc = kc; q.splits = 1;
      if (plan_smem(p, q) > 200 * 1024 || (size_t)kc * (p.maps * p.kdp + p.rotp + 4 + (p.shared ? 0 : p.vdp)) + (size_t)R * (p.kdp + p.rotp) < (size_t)R * p.vdp) continue;
      const uint32_t ctas = B * p.G * q.subs * p.T, room = ctas >= 592 ? 1 : 592 / ctas;
      q.splits = std::max(1u, std::min(std::min((most + kc - 1) / kc, room), 32u));
      *pl = q;
      found = true;
      if ((uint64_t)ctas * q.splits >= 96) return true;
      break;
    }
  }
  return found;
}

__global__ void __launch_bounds__(32) diff_lambda_kernel(const float* a1, const float* b1, const float* a2, const float* b2, uint32_t n, float add, float* out) {
  float s1 = 0.0f, s2 = 0.0f;
  for (uint32_t i = threadIdx.x; i < n; i += 32) { s1 = fmaf(a1[i], b1[i], s1); s2 = fmaf(a2[i], b2[i], s2); }
  s1 = warp_sum(s1);
  s2 = warp_sum(s2);
  if (threadIdx.x == 0) *out = expf(s1) - expf(s2) + add;
}

}  // namespace

size_t ruai_attn_span_scratch(const SpanParams& p, uint32_t B, size_t* counters) {
  Plan pl;
  *counters = 0;
  if (!make_plan(p, B, &pl) || pl.splits == 1) return 0;
  *counters = (size_t)B * p.G * pl.subs * p.T;
  return *counters * pl.splits * pl.rc * p.maps * (p.vdp + 4) * sizeof(float);
}

int ruai_span_append(ruai_ctx* c, const SpanParams& p, uint32_t B) {
  const uint32_t rows = B * p.T, per = p.G * (p.rep * p.maps + p.maps + (p.shared ? 0 : 1));
  if ((uint64_t)rows * per > 0xFFFFFFF0ull) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "a step of %u tokens is too large", rows);
  RUAI_CUDA(c, ruai_launch(c, span_append_kernel, dim3((rows * per + kWarps - 1) / kWarps), dim3(kThreads), 0, true, p, rows));
  return RUAI_OK;
}

int ruai_attn_span(ruai_ctx* c, const SpanParams& p, uint32_t B) {
  if (p.maps < 1 || p.maps > 2) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "%u score maps per head (1 or 2)", p.maps);
  if (p.maps == 2 && (p.rot || p.shared || p.sink)) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "two score maps with a rotated part, shared values or a sink");
  if (p.shared && p.vdp > p.kdp) return ruai_fail(c, RUAI_ERR_SHAPE, "values of %u elements at the front of keys of %u", p.vd, p.kd);
  const bool fuse = p.T == 1;
  if (!fuse) {
    RUAI_TRY(ruai_span_append(c, p, B));
    if (!p.rot && !p.shared && !p.sink && !p.gate) {
      AttnParams ap = {};
      ap.q = p.q; ap.q_ld = p.G * p.rep * p.maps * p.kdp; ap.kcache = p.kcache; ap.vcache = p.vcache; ap.len = p.len; ap.T = p.T; ap.KV = p.G;
      ap.hd = p.kdp; ap.vd = p.vdp; ap.vd_out = p.vd; ap.maps = p.maps; ap.window = p.window; ap.keep = p.keep; ap.cap = p.cap; ap.scale = p.scale;
      ap.lambda = p.lambda; ap.out_scale = p.out_scale; ap.eps = p.eps;
      ap.out = (float*)p.out; ap.out_ld = p.out_ld; ap.out_dtype = p.out_dtype; ap.status = p.status;
      const int took = ruai_attention_prefill(c, ap, B, p.rep);
      if (took < 0) return RUAI_ERR_CUDA;
      if (took) return RUAI_OK;
    }
  }
  Plan pl;
  if (!make_plan(p, B, &pl)) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "attention heads of %u maps x %u keys, %u values are too large", p.maps, p.kd + p.rot, p.vd);
  if (p.T > 65535) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "a step of %u tokens is too large for this head shape", p.T);
  static bool attr_done[64] = {};
  if (!attr_done[c->ordinal & 63]) {
    for (auto k : {span_attention_kernel<true, false>, span_attention_kernel<false, false>, span_attention_kernel<true, true>, span_attention_kernel<false, true>})
      RUAI_CUDA(c, cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr_done[c->ordinal & 63] = true;
  }
  const dim3 grid(B * p.G * pl.subs, p.T, pl.splits);
  const size_t smem = plan_smem(p, pl);
  auto kernel = p.shared ? (fuse ? span_attention_kernel<true, true> : span_attention_kernel<false, true>)
                         : (fuse ? span_attention_kernel<true, false> : span_attention_kernel<false, false>);
  RUAI_CUDA(c, ruai_launch(c, kernel, grid, dim3(kThreads), smem, true, p, pl));
  return RUAI_OK;
}

int ruai_diff_lambda(ruai_ctx* c, const float* a1, const float* b1, const float* a2, const float* b2, uint32_t n, float add, float* out) {
  diff_lambda_kernel<<<1, 32, 0, c->stream>>>(a1, b1, a2, b2, n, add, out);
  RUAI_CUDA(c, cudaGetLastError());
  return RUAI_OK;
}
