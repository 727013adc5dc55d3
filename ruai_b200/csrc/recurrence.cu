// Linear attention with a matrix state per head and a per-channel decay, in f32: one parameterised recurrence serves
// every mixer of the kind (with a bonus for the current token, or with the forget gate as the complement of the key).
//
//   recurrence_step_kernel  one token: a CTA per (sequence, head); the state streams through once, coalesced along the
//                           value columns, with the decay's low-rank projection, the head's norm and the gate fused.
//   recurrence_scan_kernel  many tokens: the columns of the state never meet, so a half warp owns one, two or four value
//                           columns (its 16 lanes share the key channels, the state stays in registers) and walks the
//                           tokens; keys, decays and reads of the next block of tokens arrive by cp.async meanwhile.
//                           The sums over the lanes are taken for four tokens at once: every exchange halves what a
//                           lane still holds.
//   head_norm_kernel        the scan's outputs: per (token, head) division by the root mean square, weight, gate.
#include "recurrence.cuh"

#include "scan.cuh"

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  return v;
}

// ---- one token ------------------------------------------------------------------------------------------

constexpr int kSThreads = 512, kSWarps = kSThreads / 32;
constexpr int kSHold = 32;     // state elements a thread holds in registers, requested ahead of the dependency wait
constexpr int kSRows = 4;      // rows of the decay projection per warp that are requested ahead of it too (two elements a lane)

__global__ void __launch_bounds__(kSThreads) recurrence_step_kernel(const RecurrenceParams p) {
  extern __shared__ float sm[];
  const uint32_t h = blockIdx.x, b = blockIdx.y, dk = p.dk, dv = p.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *r = sm, *k = r + dk, *w = k + dk, *us = w + dk, *o = us + dk, *red = o + dv, *part = red + 32;  // part [groups][vc]
  const uint32_t vc = min((uint32_t)kSThreads, (dv + 31u) & ~31u), groups = kSThreads / vc, per = (dk + groups - 1) / groups;
  const uint32_t kg = tid / vc, col0 = tid % vc, ka = min(dk, kg * per), kb = min(dk, ka + per);
  const bool worker = kg < groups;
  float* S = p.state + ((size_t)b * p.H + h) * dk * dv;
  // The state and the position are earlier steps' work and the weights are constant: all of it may be read while the
  // predecessor still runs.
  const bool fresh = __ldcg(p.len) == 0;
  float hold[kSHold];
  auto hold_state = [&](uint32_t c, uint32_t i0) {
#pragma unroll
    for (int q = 0; q < kSHold; ++q) {
      const uint32_t i = i0 + q;
      hold[q] = (worker && c < dv && i < kb && !fresh) ? __ldcg(S + (size_t)i * dv + c) : 0.0f;
    }
  };
  hold_state(col0, ka);
  float w2v[kSRows][2];
  const int w2_type = p.w2_bits == 16 ? RUAI_BF16 : RUAI_F32;
  if (!p.w) {
#pragma unroll
    for (int q = 0; q < kSRows; ++q) {
      const uint32_t i = warp + kSWarps * q;
#pragma unroll
      for (int e = 0; e < 2; ++e)
        w2v[q][e] = (i < dk && lane + 32 * e < p.rank) ? load_as_f32(p.w2, w2_type, ((size_t)h * dk + i) * p.w2_ld + lane + 32 * e) : 0.0f;
    }
  }
  float w0v[kSRows];
#pragma unroll
  for (int q = 0; q < kSRows; ++q) {
    const uint32_t i = warp + kSWarps * q;
    w0v[q] = (!p.w && i < dk) ? p.w0[(size_t)h * dk + i] : 0.0f;
  }
  if (p.u && tid < dk) us[tid] = p.u[(size_t)h * dk + tid];  // dk <= kSThreads
  const float norm0 = tid < dv ? p.norm[p.norm_per_head ? h * dv + tid : tid] : 0.0f;
  grid_dependency_wait();
  grid_launch_dependents();
  // everything the predecessor left, requested together
  const float* vrow = p.v + (size_t)b * p.ld_v + (size_t)h * dv;
  const float rv = tid < dk ? p.r[(size_t)b * p.ld_r + h * dk + tid] : 0.0f;
  const float wv = (p.w && tid < dk) ? p.w[(size_t)b * p.ld_w + h * dk + tid] : 0.0f;
  const float kv0 = (p.k && tid < dk) ? p.k[(size_t)b * p.ld_k + h * dk + tid] : 1.0f - wv;
  const float v0 = col0 < dv ? vrow[col0] : 0.0f;
  const float gate0 = (p.gate && tid < dv) ? p.gate[(size_t)b * p.ld_gate + (size_t)h * dv + tid] : 1.0f;
  if (tid < dk) {
    r[tid] = rv;
    if (p.w) w[tid] = wv;
    if (p.w || p.k) k[tid] = kv0;
  }
  if (!p.w) {
    float tv[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) tv[e] = lane + 32 * e < p.rank ? load_as_f32(p.t, p.t_dtype, (size_t)b * p.ld_t + lane + 32 * e) : 0.0f;
    auto put = [&](uint32_t i, float a, float w0) {
      a = warp_sum(a);
      if (lane == 0) {
        const float f = expf(-expf(a + w0));
        w[i] = f;
        if (!p.k) k[i] = 1.0f - f;
      }
    };
    auto rest = [&](uint32_t i, uint32_t e0, float a) {
      for (uint32_t e = e0; e < p.rank; e += 32)
        a = fmaf(load_as_f32(p.w2, w2_type, ((size_t)h * dk + i) * p.w2_ld + e), load_as_f32(p.t, p.t_dtype, (size_t)b * p.ld_t + e), a);
      return a;
    };
#pragma unroll
    for (int q = 0; q < kSRows; ++q) {
      const uint32_t i = warp + kSWarps * q;
      if (i < dk) put(i, rest(i, lane + 64, fmaf(w2v[q][0], tv[0], w2v[q][1] * tv[1])), w0v[q]);
    }
    for (uint32_t i = warp + kSWarps * kSRows; i < dk; i += kSWarps) put(i, rest(i, lane, 0.0f), p.w0[(size_t)h * dk + i]);
  }
  __syncthreads();
  const bool bonus = p.u != nullptr;
  for (uint32_t c0 = 0; c0 < dv; c0 += vc) {
    const uint32_t c = c0 + col0;
    const float v = c0 == 0 ? v0 : (c < dv ? vrow[c] : 0.0f);
    float acc = 0.0f;
    for (uint32_t i0 = ka; i0 < kb; i0 += kSHold) {
      if (c0 > 0 || i0 > ka) hold_state(c, i0);
#pragma unroll
      for (int q = 0; q < kSHold; ++q) {
        const uint32_t i = min(i0 + q, dk - 1);
        const float s = hold[q], kv = k[i] * v, sn = fmaf(w[i], s, kv), add = r[i] * (bonus ? fmaf(us[i], kv, s) : sn);
        if (i0 + q < kb) acc += add;
        hold[q] = sn;
      }
      if (worker && c < dv) {
#pragma unroll
        for (int q = 0; q < kSHold; ++q)
          if (i0 + q < kb) S[(size_t)(i0 + q) * dv + c] = hold[q];
      }
    }
    if (worker) part[kg * vc + col0] = acc;
    __syncthreads();
    if (kg == 0 && c < dv) {
      float t = 0.0f;
      for (uint32_t g = 0; g < groups; ++g) t += part[g * vc + col0];
      o[c] = t;
    }
    __syncthreads();
  }
  float ss = 0.0f;
  for (uint32_t c = tid; c < dv; c += kSThreads) ss = fmaf(o[c], o[c], ss);
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = 0.0f;
  for (int i = 0; i < kSWarps; ++i) ss += red[i];
  const float rs = 1.0f / sqrtf(ss / (float)dv + p.eps);
  for (uint32_t c = tid; c < dv; c += kSThreads) {
    float y = o[c] * rs * (c < kSThreads ? norm0 : p.norm[p.norm_per_head ? h * dv + c : c]);
    if (p.gate) y *= c < kSThreads ? gate0 : p.gate[(size_t)b * p.ld_gate + (size_t)h * dv + c];
    store_from_f32(p.out, p.out_dtype, (size_t)b * p.out_ld + (size_t)h * dv + c, y);
  }
}

// ---- many tokens ---------------------------------------------------------------------------------------------

constexpr int kCThreads = 256, kLanes = 16, kOwners = kCThreads / kLanes;  // half warps per CTA

// grid (blocks of kOwners * C value columns, heads, sequences); a half warp owns C columns, KPL key channels per lane; a
// block of tokens holds tc of them (a multiple of 4).  Reading keys, decays and receptances from shared memory is what
// bounds the kernel, hence several columns per thread.
// Shared memory: two buffers of [tc][3 (r, k, w)][16 KPL] and [tc][kOwners * C] values.
template <int KPL, int C, bool BONUS>
__global__ void __launch_bounds__(kCThreads) recurrence_scan_kernel(const RecurrenceParams p, uint32_t tc, int vec, int vec_v) {
  extern __shared__ __align__(16) float sm[];
  constexpr uint32_t kRow = kLanes * KPL, kCols = kOwners * C;
  constexpr int kAhead = KPL == 4 ? 4 : KPL == 8 ? 2 : 1;
  const uint32_t h = blockIdx.y, b = blockIdx.z, dk = p.dk, dv = p.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t l = tid & (kLanes - 1), cl = tid / kLanes * C, cb = blockIdx.x * kCols, T = p.T;
  const uint32_t buf_floats = tc * (3 * kRow + kCols);
  // channels past dk stay zero: they add nothing to any sum
  for (uint32_t i = tid; i < 2 * buf_floats; i += kCThreads) sm[i] = 0.0f;
  __syncthreads();
  grid_dependency_wait();
  grid_launch_dependents();
  // A warp fetches every (kCThreads / 32)-th token; its lanes' addresses only ever move on by that many rows.
  constexpr uint32_t kStep = kCThreads / 32;
  const size_t row0 = (size_t)b * T + warp;
  const uint32_t el = vec ? 4 * lane : lane, evl = vec_v ? 4 * lane : lane;
  const float *pr = p.r + row0 * p.ld_r + h * dk + el, *pw = p.w + row0 * p.ld_w + h * dk + el;
  const float* pk = BONUS ? p.k + row0 * p.ld_k + h * dk + el : nullptr;
  const float* pv = p.v + row0 * p.ld_v + (size_t)h * dv + cb + evl;
  const size_t step_r = (size_t)kStep * p.ld_r, step_k = (size_t)kStep * p.ld_k, step_w = (size_t)kStep * p.ld_w, step_v = (size_t)kStep * p.ld_v;
  const bool v_mine = evl < kCols && cb + evl < dv;
  const uint32_t de = vec ? 128 : 32;
  auto fetch = [&](uint32_t t0, uint32_t buf) {  // blocks of tokens in order
    float* d = sm + buf * buf_floats + warp * 3 * kRow + el;
    float* dv_ = sm + buf * buf_floats + tc * 3 * kRow + warp * kCols + evl;
    const uint32_t n = min(tc, T - t0);
    for (uint32_t t = warp; t < n; t += kStep) {
      if (vec) {
        for (uint32_t e = 0; el + e < dk; e += de) {
          cp_async16(d + e, pr + e);
          if (BONUS) cp_async16(d + kRow + e, pk + e);
          cp_async16(d + 2 * kRow + e, pw + e);
        }
      } else {
        for (uint32_t e = 0; el + e < dk; e += de) {
          cp_async4(d + e, pr + e);
          if (BONUS) cp_async4(d + kRow + e, pk + e);
          cp_async4(d + 2 * kRow + e, pw + e);
        }
      }
      if (v_mine) {
        if (vec_v) cp_async16(dv_, pv);
        else cp_async4(dv_, pv);
      }
      pr += step_r; pw += step_w; pv += step_v;
      if (BONUS) pk += step_k;
      d += kStep * 3 * kRow; dv_ += kStep * kCols;
    }
    cp_commit();
  };
  fetch(0, 0);
  f32x2 S[C][KPL / 2], u[KPL / 2];
  float* st = p.state + ((size_t)b * p.H + h) * dk * dv;
  const bool fresh = *p.len == 0;
  auto channel = [&](int i) { return 4 * (l + kLanes * (i / 4)) + i % 4; };  // a lane has channels 4 l .. 4 l + 3 of every 64
#pragma unroll
  for (int i = 0; i < KPL; i += 2) {
    const uint32_t k0 = channel(i), k1 = channel(i + 1);
    u[i / 2] = BONUS ? pack2(k0 < dk ? p.u[(size_t)h * dk + k0] : 0.0f, k1 < dk ? p.u[(size_t)h * dk + k1] : 0.0f) : 0;
#pragma unroll
    for (int j = 0; j < C; ++j) {
      const bool in = cb + cl + j < dv && !fresh;
      S[j][i / 2] = pack2(in && k0 < dk ? st[(size_t)k0 * dv + cb + cl + j] : 0.0f, in && k1 < dk ? st[(size_t)k1 * dv + cb + cl + j] : 0.0f);
    }
  }
  uint32_t buf = 0;
  for (uint32_t t0 = 0; t0 < T; t0 += tc, buf ^= 1) {
    if (t0 + tc < T) { fetch(t0 + tc, buf ^ 1); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    const float* s = sm + buf * buf_floats;
    const float* sv = s + tc * 3 * kRow;
    const uint32_t n = min(tc, T - t0);
    // What a token brings to this lane, and its step.  Several tokens' values are requested ahead of the first one's step:
    // the latency of shared memory would otherwise be paid token by token.
    struct In { f32x2 r[KPL / 2], k[KPL / 2], w[KPL / 2]; float v[C]; };
    auto load = [&](uint32_t t, In& x) {
#pragma unroll
      for (int q = 0; q < KPL / 4; ++q) {
        const float* d = s + t * 3 * kRow + 4 * (l + kLanes * q);
        const ulonglong2 r4 = *reinterpret_cast<const ulonglong2*>(d), w4 = *reinterpret_cast<const ulonglong2*>(d + 2 * kRow);
        x.r[2 * q] = r4.x; x.r[2 * q + 1] = r4.y;
        x.w[2 * q] = w4.x; x.w[2 * q + 1] = w4.y;
        if constexpr (BONUS) {
          const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(d + kRow);
          x.k[2 * q] = k4.x; x.k[2 * q + 1] = k4.y;
        } else {
          const f32x2 one = pack2(1.0f, 1.0f), minus = pack2(-1.0f, -1.0f);
          x.k[2 * q] = fma2(w4.x, minus, one); x.k[2 * q + 1] = fma2(w4.y, minus, one);
        }
      }
      if constexpr (C == 4) { const float4 v = *reinterpret_cast<const float4*>(sv + t * kCols + cl); x.v[0] = v.x; x.v[1] = v.y; x.v[2] = v.z; x.v[3] = v.w; }
      else if constexpr (C == 2) { const float2 v = *reinterpret_cast<const float2*>(sv + t * kCols + cl); x.v[0] = v.x; x.v[1] = v.y; }
      else x.v[0] = sv[t * kCols + cl];
    };
    auto step = [&](const In& x, float (&o)[C]) {
#pragma unroll
      for (int j = 0; j < C; ++j) {
        const f32x2 vv = pack2(x.v[j], x.v[j]);
        f32x2 part = 0;  // two zeros
#pragma unroll
        for (int i = 0; i < KPL / 2; ++i) {
          const f32x2 kv = mul2(x.k[i], vv), old = S[j][i];
          S[j][i] = fma2(x.w[i], old, kv);
          part = fma2(x.r[i], BONUS ? fma2(u[i], kv, old) : S[j][i], part);
        }
        const float2 h2 = unpack2(part);
        o[j] = h2.x + h2.y;
      }
    };
    const size_t orow = (size_t)p.H * dv;
    float* out = p.o + ((size_t)b * T + t0) * orow + (size_t)h * dv + cb + cl;
    uint32_t t = 0;
    for (; t + 4 <= n; t += 4) {
      constexpr int N = 4 * C;  // partial sums of four tokens: every exchange halves what a lane holds
      float z[N];
#pragma unroll
      for (int q0 = 0; q0 < 4; q0 += kAhead) {
        In x[kAhead];
#pragma unroll
        for (int q = 0; q < kAhead; ++q) load(t + q0 + q, x[q]);
#pragma unroll
        for (int q = 0; q < kAhead; ++q) {
          float o[C];
          step(x[q], o);
#pragma unroll
          for (int j = 0; j < C; ++j) z[(q0 + q) * C + j] = o[j];
        }
      }
      uint32_t idx = 0;
#pragma unroll
      for (int step = 0; step < 4; ++step) {
        const int have = N >> step;
        const uint32_t bit = 1u << step;
        if (have > 1) {
          const bool hi = l & bit;
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
      const uint32_t j = idx % C;
      if (l < (uint32_t)N && cb + cl + j < dv) out[(size_t)(t + idx / C) * orow + j] = z[0];
    }
    for (; t < n; ++t) {
      float z[C];
      In x;
      load(t, x);
      step(x, z);
#pragma unroll
      for (int j = 0; j < C; ++j) {
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) z[j] += __shfl_xor_sync(0xFFFFFFFFu, z[j], o);
        if (l == 0 && cb + cl + j < dv) out[(size_t)t * orow + j] = z[j];
      }
    }
    __syncthreads();  // the buffer may be refilled
  }
#pragma unroll
  for (int i = 0; i < KPL; i += 2) {
    const uint32_t k0 = channel(i), k1 = channel(i + 1);
#pragma unroll
    for (int j = 0; j < C; ++j) {
      const float2 v = unpack2(S[j][i / 2]);
      if (cb + cl + j < dv && k0 < dk) st[(size_t)k0 * dv + cb + cl + j] = v.x;
      if (cb + cl + j < dv && k1 < dk) st[(size_t)k1 * dv + cb + cl + j] = v.y;
    }
  }
}

// One warp per (token, head).
__global__ void __launch_bounds__(256) head_norm_kernel(const RecurrenceParams p, uint32_t rows) {
  grid_dependency_wait();
  grid_launch_dependents();
  const uint32_t lane = threadIdx.x & 31, i = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), dv = p.dv;
  if (i >= rows * p.H) return;
  const uint32_t row = i / p.H, h = i % p.H;
  const float* o = p.o + (size_t)row * p.H * dv + (size_t)h * dv;
  float ss = 0.0f;
  for (uint32_t c = lane; c < dv; c += 32) ss = fmaf(o[c], o[c], ss);
  ss = warp_sum(ss);
  const float rs = 1.0f / sqrtf(ss / (float)dv + p.eps);
  for (uint32_t c = lane; c < dv; c += 32) {
    float y = o[c] * rs * p.norm[p.norm_per_head ? h * dv + c : c];
    if (p.gate) y *= p.gate[(size_t)row * p.ld_gate + (size_t)h * dv + c];
    store_from_f32(p.out, p.out_dtype, (size_t)row * p.out_ld + (size_t)h * dv + c, y);
  }
}

template <int KPL, int C, bool BONUS>
cudaError_t launch_scan(ruai_ctx* c, const RecurrenceParams& p, uint32_t B) {
  static bool attr_done[64] = {};
  if (!attr_done[c->ordinal & 63]) {
    cudaError_t e = cudaFuncSetAttribute(recurrence_scan_kernel<KPL, C, BONUS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return e;
    attr_done[c->ordinal & 63] = true;
  }
  constexpr uint32_t kCols = kOwners * C;
  const uint32_t tc = KPL <= 4 ? 32 : 16;
  const size_t smem = 2 * (size_t)tc * (3 * kLanes * KPL + kCols) * sizeof(float);
  auto al = [](const float* q, uint32_t ld) { return !q || ((uintptr_t)q % 16 == 0 && ld % 4 == 0); };
  const int vec = p.dk % 4 == 0 && al(p.r, p.ld_r) && al(p.k, p.ld_k) && al(p.w, p.ld_w) ? 1 : 0;
  const int vec_v = p.dv % 4 == 0 && al(p.v, p.ld_v) ? 1 : 0;
  const dim3 grid((p.dv + kCols - 1) / kCols, p.H, B);
  return ruai_launch(c, recurrence_scan_kernel<KPL, C, BONUS>, grid, dim3(kCThreads), smem, true, p, tc, vec, vec_v);
}
template <int KPL, bool BONUS>
cudaError_t columns_scan(ruai_ctx* c, const RecurrenceParams& p, uint32_t B) {
  // as many columns per thread as leave most SMs a CTA
  auto ctas = [&](uint32_t cols) { return (uint64_t)((p.dv + kOwners * cols - 1) / (kOwners * cols)) * p.H * B; };
  const uint64_t enough = (uint64_t)c->sm_count * 3 / 4;
  if constexpr (KPL <= 8)
    if (ctas(4) >= enough) return launch_scan<KPL, 4, BONUS>(c, p, B);
  if (ctas(2) >= enough) return launch_scan<KPL, 2, BONUS>(c, p, B);
  return launch_scan<KPL, 1, BONUS>(c, p, B);
}
template <bool BONUS>
cudaError_t dispatch_scan(ruai_ctx* c, const RecurrenceParams& p, uint32_t B) {
  if (p.dk <= 64) return columns_scan<4, BONUS>(c, p, B);
  if (p.dk <= 128) return columns_scan<8, BONUS>(c, p, B);
  return columns_scan<16, BONUS>(c, p, B);
}

}  // namespace

int ruai_recurrence(ruai_ctx* c, const RecurrenceParams& p, uint32_t B) {
  if (p.dk == 0 || p.dv == 0 || p.dk > 256 || p.dv > 4096) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "recurrent head of %u x %u (at most 256 x 4096)", p.dk, p.dv);
  if (p.T == 1) {
    const size_t smem = (4 * (size_t)p.dk + p.dv + 32 + kSThreads) * sizeof(float);
    RUAI_CUDA(c, ruai_launch(c, recurrence_step_kernel, dim3(p.H, B), dim3(kSThreads), smem, true, p));
    return RUAI_OK;
  }
  if (!p.w || (p.u != nullptr) != (p.k != nullptr)) return ruai_fail(c, RUAI_ERR_ARG, "the scan needs its decays, and keys exactly with a bonus");
  cudaError_t e = p.u ? dispatch_scan<true>(c, p, B) : dispatch_scan<false>(c, p, B);
  if (e != cudaSuccess) return ruai_fail(c, RUAI_ERR_CUDA, "recurrence launch: %s", cudaGetErrorString(e));
  return ruai_head_norm(c, p, B * p.T);
}

int ruai_head_norm(ruai_ctx* c, const RecurrenceParams& p, uint32_t rows) {
  RUAI_CUDA(c, ruai_launch(c, head_norm_kernel, dim3((rows * p.H + 7) / 8), dim3(256), 0, true, p, rows));
  return RUAI_OK;
}
