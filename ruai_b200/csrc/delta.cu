// Gated delta rule (see delta.cuh), in f32: the state decays, its answer to the key moves towards the value, the query reads.
//
//   delta_step_kernel   one token: a CTA per (sequence, head) does all of it, convolutions included; the state streams
//                       through registers once where it fits.  q^T S of the new state is decay q^T S + (q k) u, so both
//                       products with the old state are taken in one pass.
//   delta_conv_kernel   many tokens: convolutions, silu, unit vectors, decays and q k: a warp per (head or block of value
//                       channels, four tokens), each input read once per warp.
//   conv_history_kernel the last inputs of the convolutions, for the next step.
//   delta_scan_kernel   the columns of the state never meet: a half warp owns one, two or four value columns (its 16 lanes
//                       share the key channels) and walks the tokens, whose rows arrive by cp.async in blocks.
// Then head_norm_kernel (recurrence.cu).
#include "delta.cuh"

#include <algorithm>

#include "recurrence.cuh"
#include "scan.cuh"

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  return v;
}
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float decay_of(float a_log, float a) { return expf(-expf(a_log) * softplus(a)); }

// ---- one token ------------------------------------------------------------------------------------------

constexpr int kSThreads = 512, kSWarps = kSThreads / 32;
constexpr int kSHold = 32;  // state elements a thread holds in registers, requested ahead of the dependency wait

template <int N>
__global__ void __launch_bounds__(kSThreads) delta_step_kernel(const DeltaParams p) {
  extern __shared__ float sm[];
  const uint32_t h = blockIdx.x, b = blockIdx.y, dk = p.dk, dv = p.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t rep = p.H / p.G, g = h / rep, C = 2 * p.G * dk + p.H * dv, nch = 2 * dk + dv;
  float *ch = sm, *q = ch, *k = q + dk, *v = k + dk, *o = ch + nch, *red = o + dv, *pp = red + 32;  // pp [2][groups][vc]
  __shared__ float s_unit[3];
  const uint32_t vc = min((uint32_t)kSThreads, (dv + 31u) & ~31u), groups = kSThreads / vc, per = (dk + groups - 1) / groups;
  const uint32_t kg = tid / vc, col0 = tid % vc, ka = min(dk, kg * per), kb = min(dk, ka + per);
  const bool worker = kg < groups;
  float* S = p.state + ((size_t)b * p.H + h) * dk * dv;
  const uint32_t pos = (uint32_t)__ldcg(p.len);
  const bool fresh = pos == 0;
  float hold[kSHold];
  auto load_state = [&](uint32_t c, uint32_t i0) {
#pragma unroll
    for (int e = 0; e < kSHold; ++e) {
      const uint32_t i = i0 + e;
      hold[e] = (worker && c < dv && i < kb && !fresh) ? __ldcg(S + (size_t)i * dv + c) : 0.0f;
    }
  };
  load_state(col0, ka);
  // a channel of this head: its raw input, weights and place in the history
  struct Place { const float *x, *w; uint32_t at; };
  auto place = [&](uint32_t c) {
    Place r;
    if (c < dk) r = {p.q + (size_t)b * p.ld_q + g * dk + c, p.conv_q + (size_t)(g * dk + c) * p.taps, g * dk + c};
    else if (c < 2 * dk) r = {p.k + (size_t)b * p.ld_k + g * dk + c - dk, p.conv_k + (size_t)(g * dk + c - dk) * p.taps, (p.G + g) * dk + c - dk};
    else r = {p.v + (size_t)b * p.ld_v + (size_t)h * dv + c - 2 * dk, p.conv_v + ((size_t)h * dv + c - 2 * dk) * p.taps, 2 * p.G * dk + h * dv + c - 2 * dk};
    return r;
  };
  float* hist = p.history + (size_t)b * p.taps * C;
  // earlier inputs' part of a channel's convolution
  auto past_part = [&](const Place& r) {
    float s = 0.0f;
#pragma unroll
    for (int j = 1; j < N; ++j)
      if ((uint32_t)j < p.taps && (uint32_t)j <= pos) s = fmaf(r.w[p.taps - 1 - j], __ldcg(hist + (size_t)((pos - j) % p.taps) * C + r.at), s);
    return s;
  };
  const Place mine = place(min(tid, nch - 1));
  const float part0 = tid < nch ? past_part(mine) : 0.0f, w0 = mine.w[p.taps - 1];
  const float norm0 = tid < dv ? p.norm[tid] : 0.0f, a_log = p.a_log[h];
  grid_dependency_wait();
  grid_launch_dependents();
  const float gate0 = (p.gate && tid < dv) ? p.gate[(size_t)b * p.ld_gate + (size_t)h * dv + tid] : 1.0f;
  const float a = p.a[(size_t)b * p.ld_a + h], beta = p.beta[(size_t)b * p.ld_beta + h];
  for (uint32_t c = tid; c < nch; c += kSThreads) {
    const Place r = c == tid ? mine : place(c);
    const float x = *r.x;
    ch[c] = silu(fmaf(c == tid ? w0 : r.w[p.taps - 1], x, c == tid ? part0 : past_part(r)));
    if (c >= 2 * dk || h % rep == 0) hist[(size_t)(pos % p.taps) * C + r.at] = x;
  }
  const float decay = decay_of(a_log, a);
  __syncthreads();
  if (warp < 3) {
    const float *x = warp == 1 ? k : q, *y = warp == 0 ? q : k;
    float s = 0.0f;
    for (uint32_t i = lane; i < dk; i += 32) s = fmaf(x[i], y[i], s);
    s = warp_sum(s);
    if (lane == 0) s_unit[warp] = warp == 2 ? s : 1.0f / sqrtf(s + p.unit_eps);
  }
  __syncthreads();
  const float rq = s_unit[0] * p.q_scale, rk = s_unit[1], qk = s_unit[2] * rq * rk;
  for (uint32_t c0 = 0; c0 < dv; c0 += vc) {
    const uint32_t c = c0 + col0;
    float sk = 0.0f, sq = 0.0f;
    for (uint32_t i0 = ka; i0 < kb; i0 += kSHold) {
      if (c0 > 0 || i0 > ka) load_state(c, i0);
#pragma unroll
      for (int e = 0; e < kSHold; ++e) {
        const uint32_t i = min(i0 + e, dk - 1);
        if (i0 + e < kb) { sk = fmaf(hold[e], k[i], sk); sq = fmaf(hold[e], q[i], sq); }
      }
    }
    if (worker) { pp[kg * vc + col0] = sk; pp[(groups + kg) * vc + col0] = sq; }
    __syncthreads();
    if (worker && c < dv) {
      sk = 0.0f; sq = 0.0f;
      for (uint32_t e = 0; e < groups; ++e) { sk += pp[e * vc + col0]; sq += pp[(groups + e) * vc + col0]; }
      const float u = beta * (v[c] - decay * rk * sk);
      if (kg == 0) o[c] = fmaf(qk, u, decay * rq * sq);
      const float uk = u * rk;
      const bool one = kb - ka <= (uint32_t)kSHold;  // what the registers hold is the whole of this thread's share
      for (uint32_t i0 = ka; i0 < kb; i0 += kSHold) {
        if (!one) load_state(c, i0);
#pragma unroll
        for (int e = 0; e < kSHold; ++e)
          if (i0 + e < kb) S[(size_t)(i0 + e) * dv + c] = fmaf(k[i0 + e], uk, decay * hold[e]);
      }
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
    float y = o[c] * rs * (c == tid ? norm0 : p.norm[c]);
    if (p.gate) y *= c == tid ? gate0 : p.gate[(size_t)b * p.ld_gate + (size_t)h * dv + c];
    store_from_f32(p.out, p.out_dtype, (size_t)b * p.out_ld + (size_t)h * dv + c, y);
  }
}

// ---- many tokens: what enters the recurrence -----------------------------------------------------------------

struct Work {  // rows of tokens; channels past dk (up to dkp) are zero
  float *q, *k, *v, *sc, *o;  // [G * dkp], [G * dkp], [H * dvp], [H][decay, beta, q k, -], [H * dv]
  uint32_t dkp, dvp;
};
__host__ __device__ inline uint32_t up4(uint32_t v) { return (v + 3) & ~3u; }
Work work_of(const DeltaParams& p, uint32_t rows) {
  Work w;
  w.dkp = up4(p.dk); w.dvp = up4(p.dv);
  w.q = p.work;
  w.k = w.q + (size_t)rows * p.G * w.dkp;
  w.v = w.k + (size_t)rows * p.G * w.dkp;
  w.sc = w.v + (size_t)rows * p.H * w.dvp;
  w.o = w.sc + (size_t)rows * p.H * 4;
  return w;
}

constexpr int kTT = 4;  // tokens per warp
constexpr uint32_t kValueBlock = 128;

// items: (sequence, block of kTT tokens, unit); units: G pairs of q and k heads, then blocks of value channels
template <int N, int CH>
__global__ void __launch_bounds__(256) delta_conv_kernel(const DeltaParams p, const Work w, uint32_t items, uint32_t units, uint32_t tiles) {
  grid_dependency_wait();
  grid_launch_dependents();
  const uint32_t item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= items) return;
  const uint32_t unit = item % units, t0 = item / units % tiles * kTT, b = item / units / tiles;
  const uint32_t dk = p.dk, dv = p.dv, C = 2 * p.G * dk + p.H * dv, past = (uint32_t)*p.len, nt = min((uint32_t)kTT, p.T - t0);
  const float* hist = p.history + (size_t)b * p.taps * C;
  auto conv = [&](const float* x, uint32_t ld, const float* taps, uint32_t at, float (&y)[kTT]) {
    float tw[N], in[kTT + N - 1];
#pragma unroll
    for (int j = 0; j < N; ++j) tw[j] = (uint32_t)(N - 1 - j) < p.taps ? taps[p.taps - (N - j)] : 0.0f;
#pragma unroll
    for (int i = 0; i < kTT + N - 1; ++i) {
      const int s = (int)t0 - (N - 1) + i;
      if (s >= 0) in[i] = s < (int)p.T ? x[((size_t)b * p.T + s) * ld] : 0.0f;
      else in[i] = ((uint32_t)-s < p.taps && (uint32_t)-s <= past) ? hist[(size_t)((past + s) % p.taps) * C + at] : 0.0f;
    }
#pragma unroll
    for (int t = 0; t < kTT; ++t) {
      float s = 0.0f;
#pragma unroll
      for (int j = 0; j < N; ++j) s = fmaf(tw[j], in[t + j], s);
      y[t] = silu(s);
    }
  };
  const size_t row0 = (size_t)b * p.T + t0;
  if (unit < p.G) {
    const uint32_t g = unit, rep = p.H / p.G;
    float q[CH][kTT], k[CH][kTT], qq[kTT] = {}, kk[kTT] = {}, qk[kTT] = {};
#pragma unroll
    for (int e = 0; e < CH; ++e) {
      const uint32_t c = lane + 32 * e;
#pragma unroll
      for (int t = 0; t < kTT; ++t) { q[e][t] = 0.0f; k[e][t] = 0.0f; }
      if (c < dk) {
        const uint32_t gc = g * dk + c;
        conv(p.q + gc, p.ld_q, p.conv_q + (size_t)gc * p.taps, gc, q[e]);
        conv(p.k + gc, p.ld_k, p.conv_k + (size_t)gc * p.taps, p.G * dk + gc, k[e]);
      }
#pragma unroll
      for (int t = 0; t < kTT; ++t) { qq[t] = fmaf(q[e][t], q[e][t], qq[t]); kk[t] = fmaf(k[e][t], k[e][t], kk[t]); qk[t] = fmaf(q[e][t], k[e][t], qk[t]); }
    }
#pragma unroll
    for (int t = 0; t < kTT; ++t) {
      const float rq = p.q_scale / sqrtf(warp_sum(qq[t]) + p.unit_eps), rk = 1.0f / sqrtf(warp_sum(kk[t]) + p.unit_eps), x = warp_sum(qk[t]) * rq * rk;
      if ((uint32_t)t >= nt) break;
      const size_t row = row0 + t;
#pragma unroll
      for (int e = 0; e < CH; ++e) {
        const uint32_t c = lane + 32 * e;
        if (c < w.dkp) {
          w.q[(row * p.G + g) * w.dkp + c] = q[e][t] * rq;
          w.k[(row * p.G + g) * w.dkp + c] = k[e][t] * rk;
        }
      }
      for (uint32_t i = lane; i < rep; i += 32) {
        const uint32_t h = g * rep + i;
        reinterpret_cast<float4*>(w.sc)[row * p.H + h] = make_float4(decay_of(p.a_log[h], p.a[row * p.ld_a + h]), p.beta[row * p.ld_beta + h], x, 0.0f);
      }
    }
  } else {
    const uint32_t c0 = (unit - p.G) * kValueBlock, c1 = min(p.H * dv, c0 + kValueBlock);
    for (uint32_t c = c0 + lane; c < c1; c += 32) {
      float y[kTT];
      conv(p.v + c, p.ld_v, p.conv_v + (size_t)c * p.taps, 2 * p.G * dk + c, y);
      const uint32_t at = c / dv * w.dvp + c % dv;
#pragma unroll
      for (int t = 0; t < kTT; ++t)
        if ((uint32_t)t < nt) w.v[(row0 + t) * p.H * w.dvp + at] = y[t];
    }
  }
}

// grid (blocks of channels, the step's last min(T, taps) tokens, sequences)
__global__ void __launch_bounds__(256) conv_history_kernel(const DeltaParams p) {
  grid_dependency_wait();
  grid_launch_dependents();
  const uint32_t qk = p.G * p.dk, C = 2 * qk + p.H * p.dv, c = blockIdx.x * 256 + threadIdx.x, t = p.T - 1 - blockIdx.y, b = blockIdx.z;
  if (c >= C) return;
  const size_t row = (size_t)b * p.T + t;
  const float v = c < qk ? p.q[row * p.ld_q + c] : c < 2 * qk ? p.k[row * p.ld_k + c - qk] : p.v[row * p.ld_v + c - 2 * qk];
  p.history[((size_t)b * p.taps + ((uint32_t)*p.len + t) % p.taps) * C + c] = v;
}

// ---- many tokens: the recurrence ------------------------------------------------------------------------------

constexpr int kCThreads = 256, kLanes = 16, kOwners = kCThreads / kLanes;

// grid (blocks of kOwners * C value columns, heads, sequences).  Shared memory: two buffers of [tc][2 (q, k)][16 KPL],
// [tc][kOwners * C] values and [tc][4] numbers of the token.
template <int KPL, int C>
__global__ void __launch_bounds__(kCThreads) delta_scan_kernel(const DeltaParams p, const Work w, uint32_t tc) {
  extern __shared__ __align__(16) float sm[];
  constexpr uint32_t kRow = kLanes * KPL, kCols = kOwners * C;
  const uint32_t h = blockIdx.y, b = blockIdx.z, dk = p.dk, dv = p.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t l = tid & (kLanes - 1), cl = tid / kLanes * C, cb = blockIdx.x * kCols, T = p.T, g = h / (p.H / p.G);
  const uint32_t buf_floats = tc * (2 * kRow + kCols + 4);
  for (uint32_t i = tid; i < 2 * buf_floats; i += kCThreads) sm[i] = 0.0f;  // channels past dkp stay zero
  __syncthreads();
  grid_dependency_wait();
  grid_launch_dependents();
  auto fetch = [&](uint32_t t0, uint32_t buf) {
    float* base = sm + buf * buf_floats;
    const uint32_t n = min(tc, T - t0);
    for (uint32_t t = warp; t < n; t += kCThreads / 32) {
      const size_t row = (size_t)b * T + t0 + t;
      const float *q = w.q + (row * p.G + g) * w.dkp, *k = w.k + (row * p.G + g) * w.dkp, *v = w.v + row * p.H * w.dvp + (size_t)h * w.dvp + cb;
      float* d = base + t * 2 * kRow;
      for (uint32_t e = 4 * lane; e < w.dkp; e += 128) {
        cp_async16(d + e, q + e);
        cp_async16(d + kRow + e, k + e);
      }
      if (4 * lane < kCols && cb + 4 * lane < w.dvp) cp_async16(base + tc * 2 * kRow + t * kCols + 4 * lane, v + 4 * lane);
      if (lane == 31) cp_async16(base + tc * (2 * kRow + kCols) + 4 * t, w.sc + (row * p.H + h) * 4);
    }
    cp_commit();
  };
  fetch(0, 0);
  f32x2 S[C][KPL / 2];
  float* st = p.state + ((size_t)b * p.H + h) * dk * dv;
  const bool fresh = *p.len == 0;
  auto channel = [&](int i) { return 4 * (l + kLanes * (i / 4)) + i % 4; };  // a lane has channels 4 l .. 4 l + 3 of every 64
#pragma unroll
  for (int i = 0; i < KPL; i += 2) {
    const uint32_t k0 = channel(i), k1 = channel(i + 1);
#pragma unroll
    for (int j = 0; j < C; ++j) {
      const bool in = cb + cl + j < dv && !fresh;
      S[j][i / 2] = pack2(in && k0 < dk ? st[(size_t)k0 * dv + cb + cl + j] : 0.0f, in && k1 < dk ? st[(size_t)k1 * dv + cb + cl + j] : 0.0f);
    }
  }
  // where the sums over the lanes end up: products with k on even lanes, with q on odd ones, column `jl`
  constexpr int kBits = C == 4 ? 2 : C == 2 ? 1 : 0;
  const uint32_t jl = C == 4 ? ((l >> 1) & 1) * 2 + ((l >> 2) & 1) : C == 2 ? (l >> 1) & 1 : 0;
  const bool writer = (l & 1) && (l >> (1 + kBits)) == 0 && cb + cl + jl < dv;
  uint32_t buf = 0;
  for (uint32_t t0 = 0; t0 < T; t0 += tc, buf ^= 1) {
    if (t0 + tc < T) { fetch(t0 + tc, buf ^ 1); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    const float* s = sm + buf * buf_floats;
    const float *sv = s + tc * 2 * kRow, *ss = sv + tc * kCols;
    const uint32_t n = min(tc, T - t0);
    struct In { f32x2 q[KPL / 2], k[KPL / 2]; float4 sc; float v; };
    auto load = [&](uint32_t t, In& x) {
#pragma unroll
      for (int e = 0; e < KPL / 4; ++e) {
        const float* d = s + t * 2 * kRow + 4 * (l + kLanes * e);
        const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(d), k4 = *reinterpret_cast<const ulonglong2*>(d + kRow);
        x.q[2 * e] = q4.x; x.q[2 * e + 1] = q4.y;
        x.k[2 * e] = k4.x; x.k[2 * e + 1] = k4.y;
      }
      x.sc = *reinterpret_cast<const float4*>(ss + 4 * t);
      x.v = sv[t * kCols + cl + jl];
    };
    const size_t orow = (size_t)p.H * dv;
    float* out = w.o + ((size_t)b * T + t0) * orow + (size_t)h * dv + cb + cl + jl;
    In x;
    load(0, x);
    for (uint32_t t = 0; t < n; ++t) {
      In nx;
      load(min(t + 1, n - 1), nx);
      float z[2 * C];
#pragma unroll
      for (int j = 0; j < C; ++j) {
        f32x2 a = 0, c = 0;
#pragma unroll
        for (int i = 0; i < KPL / 2; ++i) { a = fma2(x.k[i], S[j][i], a); c = fma2(x.q[i], S[j][i], c); }
        const float2 a2 = unpack2(a), c2 = unpack2(c);
        z[j] = a2.x + a2.y; z[C + j] = c2.x + c2.y;
      }
#pragma unroll
      for (int step = 0; step < 4; ++step) {
        const int have = 2 * C >> step;
        const uint32_t bit = 1u << step;
        if (have > 1) {
          const bool hi = l & bit;
#pragma unroll
          for (int i = 0; i < have / 2; ++i) {
            const float send = hi ? z[i] : z[i + have / 2], keep = hi ? z[i + have / 2] : z[i];
            z[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, bit);
          }
        } else {
          z[0] += __shfl_xor_sync(0xFFFFFFFFu, z[0], bit);
        }
      }
      const float decay = x.sc.x, mine = x.sc.y * (x.v - decay * z[0]);  // u of column jl, on even lanes
      float u[C];
#pragma unroll
      for (int j = 0; j < C; ++j) u[j] = __shfl_sync(0xFFFFFFFFu, mine, C == 4 ? (j >> 1) * 2 + (j & 1) * 4 : 2 * j, kLanes);
      const f32x2 dd = pack2(decay, decay);
#pragma unroll
      for (int j = 0; j < C; ++j) {
        const f32x2 uu = pack2(u[j], u[j]);
#pragma unroll
        for (int i = 0; i < KPL / 2; ++i) S[j][i] = fma2(x.k[i], uu, mul2(dd, S[j][i]));
      }
      float um = u[0];
#pragma unroll
      for (int j = 1; j < C; ++j) um = jl == (uint32_t)j ? u[j] : um;
      if (writer) out[(size_t)t * orow] = fmaf(x.sc.z, um, decay * z[0]);
      x = nx;
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

template <int KPL, int C>
cudaError_t launch_scan(ruai_ctx* c, const DeltaParams& p, const Work& w, uint32_t B) {
  static bool attr_done[64] = {};
  if (!attr_done[c->ordinal & 63]) {
    cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<KPL, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return e;
    attr_done[c->ordinal & 63] = true;
  }
  constexpr uint32_t kCols = kOwners * C;
  const uint32_t tc = KPL <= 8 ? 32 : 16;
  const size_t smem = 2 * (size_t)tc * (2 * kLanes * KPL + kCols + 4) * sizeof(float);
  return ruai_launch(c, delta_scan_kernel<KPL, C>, dim3((p.dv + kCols - 1) / kCols, p.H, B), dim3(kCThreads), smem, true, p, w, tc);
}
template <int KPL>
cudaError_t columns_scan(ruai_ctx* c, const DeltaParams& p, const Work& w, uint32_t B) {
  // as many columns per thread as leave every SM some CTAs: the tokens follow one another, so warps hide each other's waits
  auto ctas = [&](uint32_t cols) { return (uint64_t)((p.dv + kOwners * cols - 1) / (kOwners * cols)) * p.H * B; };
  const uint64_t enough = (uint64_t)c->sm_count * 3 / 2;
  if constexpr (KPL <= 8)
    if (ctas(4) >= enough) return launch_scan<KPL, 4>(c, p, w, B);
  if (ctas(2) >= enough) return launch_scan<KPL, 2>(c, p, w, B);
  return launch_scan<KPL, 1>(c, p, w, B);
}

template <int N>
cudaError_t launch_conv(ruai_ctx* c, const DeltaParams& p, const Work& w, uint32_t B) {
  const uint32_t units = p.G + (p.H * p.dv + kValueBlock - 1) / kValueBlock, tiles = (p.T + kTT - 1) / kTT, items = B * tiles * units;
  const dim3 grid((items + 7) / 8);
  return p.dk <= 128 ? ruai_launch(c, delta_conv_kernel<N, 4>, grid, dim3(256), 0, true, p, w, items, units, tiles)
                     : ruai_launch(c, delta_conv_kernel<N, 8>, grid, dim3(256), 0, true, p, w, items, units, tiles);
}

}  // namespace

size_t ruai_delta_work(const DeltaParams& p, uint32_t rows) {
  return (size_t)rows * (2 * (size_t)p.G * up4(p.dk) + (size_t)p.H * up4(p.dv) + 4 * (size_t)p.H + (size_t)p.H * p.dv);
}

int ruai_delta(ruai_ctx* c, const DeltaParams& p, uint32_t B) {
  if (!p.dk || !p.dv || p.dk > 256 || p.dv > 4096) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "recurrent head of %u x %u (at most 256 x 4096)", p.dk, p.dv);
  if (!p.taps || p.taps > (uint32_t)kConvMax) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "a convolution of %u taps (1 to %d)", p.taps, kConvMax);
  if (p.T == 1) {
    const uint32_t vc = std::min((uint32_t)kSThreads, (p.dv + 31u) & ~31u);
    const size_t smem = (2 * (size_t)p.dk + 2 * (size_t)p.dv + 32 + 2 * (size_t)(kSThreads / vc) * vc) * sizeof(float);
    RUAI_CUDA(c, p.taps <= 4 ? ruai_launch(c, delta_step_kernel<4>, dim3(p.H, B), dim3(kSThreads), smem, true, p)
                             : ruai_launch(c, delta_step_kernel<kConvMax>, dim3(p.H, B), dim3(kSThreads), smem, true, p));
    return RUAI_OK;
  }
  const uint32_t rows = B * p.T;
  if ((uint64_t)rows * (p.G + p.H * p.dv / kValueBlock + 1) > 0xFFFFFFF0ull) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "a step of %u tokens is too large", rows);
  const Work w = work_of(p, rows);
  RUAI_CUDA(c, p.taps <= 4 ? launch_conv<4>(c, p, w, B) : launch_conv<kConvMax>(c, p, w, B));
  const uint32_t C = 2 * p.G * p.dk + p.H * p.dv;
  RUAI_CUDA(c, ruai_launch(c, conv_history_kernel, dim3((C + 255) / 256, std::min(p.T, p.taps), B), dim3(256), 0, true, p));
  RUAI_CUDA(c, p.dk <= 64 ? columns_scan<4>(c, p, w, B) : p.dk <= 128 ? columns_scan<8>(c, p, w, B) : columns_scan<16>(c, p, w, B));
  RecurrenceParams r;
  r.o = w.o; r.H = p.H; r.dv = p.dv; r.eps = p.eps; r.norm = p.norm; r.gate = p.gate; r.ld_gate = p.ld_gate;
  r.out = p.out; r.out_ld = p.out_ld; r.out_dtype = p.out_dtype;
  return ruai_head_norm(c, r, rows);
}
