// Gated delta rule (see delta.cuh), in f32: the state decays, its answer to the key moves towards the value, the query reads.
//
//   delta_step_kernel   one token: a CTA per (sequence, head) does all of it, convolutions included; the state streams
//                       through registers once where it fits.  q^T S of the new state is decay q^T S + (q k) u, so both
//                       products with the old state are taken in one pass.
//   delta_conv_kernel   many tokens: convolutions, silu, unit vectors, and everything about blocks of four tokens that does
//                       not need the state: a warp per (head or block of value channels, block), each input read once.
//   conv_history_kernel the last inputs of the convolutions, for the next step.
//   delta_scan_kernel   the columns of the state never meet: a half warp owns one or two value columns (its 16 lanes share the
//                       key channels) and walks the blocks, whose rows arrive by cp.async.
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
__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.0f + expf(fminf(-z, 80.0f))); }  // the quotient is within 2 ulp
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

// The scan takes four tokens at a time.  With S the state ahead of them, g_t their decays and products over an empty range 1:
//   G_t = g_0 .. g_t,  D_ts = g_(s+1) .. g_t
//   u_t = beta_t (v_t - G_t S^T k_t - sum_(s<t) D_ts (k_t k_s) u_s)
//   o_t = G_t S^T q_t + sum_(s<=t) D_ts (q_t k_s) u_s
//   S  <- G_3 S + sum_s D_3s k_s u_s^T
// so that the products with the state wait for one another once per four tokens.  What of it does not depend on the state:
struct BlockNumbers {
  float G[4], beta[4], bG[4];  // bG = beta G
  float A[8];                  // beta_t D_ts (k_t k_s) for (t, s) = 10, 20, 21, 30, 31, 32
  float Q[4][4];               // D_ts (q_t k_s), zero for s > t
  float D[4];                  // D_3s
};
constexpr uint32_t kNumbers = sizeof(BlockNumbers) / sizeof(float);
static_assert(kNumbers == 40, "ten pieces of 16 bytes");

// Rows of tokens, each sequence's rounded up to whole blocks (the tokens past the end change nothing); channels past dk (up
// to dkp) are zero.
struct Work {
  float *q, *k, *v, *sc, *o;  // [G * dkp], [G * dkp], [H * dvp] per token, [H] BlockNumbers per block, [H * dv] per token of the step
  uint32_t dkp, dvp, Tp;
};
constexpr uint32_t kTT = 4;  // tokens per block, and per warp of the convolutions
__host__ __device__ inline uint32_t up4(uint32_t v) { return (v + 3) & ~3u; }
Work work_of(const DeltaParams& p, uint32_t B) {
  Work w;
  w.dkp = up4(p.dk); w.dvp = up4(p.dv); w.Tp = up4(p.T);
  const size_t rows = (size_t)B * w.Tp;
  w.q = p.work;
  w.k = w.q + rows * p.G * w.dkp;
  w.v = w.k + rows * p.G * w.dkp;
  w.sc = w.v + rows * p.H * w.dvp;
  w.o = w.sc + rows / kTT * p.H * kNumbers;
  return w;
}

constexpr uint32_t kValueBlock = 128;

// items: (sequence, block of kTT tokens, unit); units: G pairs of q and k heads, then blocks of value channels
template <int N, int CH>
__global__ void __launch_bounds__(256) delta_conv_kernel(const DeltaParams p, const Work w, uint32_t items, uint32_t units, uint32_t tiles) {
  grid_dependency_wait();
  grid_launch_dependents();
  const uint32_t item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= items) return;
  const uint32_t unit = item % units, tile = item / units % tiles, t0 = tile * kTT, b = item / units / tiles;
  const uint32_t dk = p.dk, dv = p.dv, C = 2 * p.G * dk + p.H * dv, past = (uint32_t)*p.len, nt = min(kTT, p.T - t0);
  const float* hist = p.history + (size_t)b * p.taps * C;
  const bool inner = t0 + 1 >= (uint32_t)N && t0 + kTT <= p.T;  // neither history nor end are near
  auto conv = [&](const float* x, uint32_t ld, const float* taps, uint32_t at, float (&y)[kTT]) {
    float tw[N], in[kTT + N - 1];
#pragma unroll
    for (int j = 0; j < N; ++j) tw[j] = (uint32_t)(N - 1 - j) < p.taps ? taps[p.taps - (N - j)] : 0.0f;
    if (inner) {
      const float* xi = x + ((size_t)b * p.T + t0 - (N - 1)) * ld;
#pragma unroll
      for (int i = 0; i < (int)kTT + N - 1; ++i) in[i] = xi[(size_t)i * ld];
    } else
#pragma unroll
    for (int i = 0; i < (int)kTT + N - 1; ++i) {
      const int s = (int)t0 - (N - 1) + i;
      if (s >= 0) in[i] = s < (int)p.T ? x[((size_t)b * p.T + s) * ld] : 0.0f;
      else in[i] = ((uint32_t)-s < p.taps && (uint32_t)-s <= past) ? hist[(size_t)((past + s) % p.taps) * C + at] : 0.0f;
    }
#pragma unroll
    for (uint32_t t = 0; t < kTT; ++t) {
      float s = 0.0f;
#pragma unroll
      for (int j = 0; j < N; ++j) s = fmaf(tw[j], in[t + j], s);
      y[t] = t < nt ? silu(s) : 0.0f;
    }
  };
  const size_t row0 = (size_t)b * w.Tp + t0, src0 = (size_t)b * p.T + t0;
  if (unit < p.G) {
    const uint32_t g = unit, rep = p.H / p.G;
    float q[CH][kTT], k[CH][kTT], qq[kTT] = {}, kk[kTT] = {};
#pragma unroll
    for (int e = 0; e < CH; ++e) {
      const uint32_t c = lane + 32 * e;
#pragma unroll
      for (uint32_t t = 0; t < kTT; ++t) { q[e][t] = 0.0f; k[e][t] = 0.0f; }
      if (c < dk) {
        const uint32_t gc = g * dk + c;
        conv(p.q + gc, p.ld_q, p.conv_q + (size_t)gc * p.taps, gc, q[e]);
        conv(p.k + gc, p.ld_k, p.conv_k + (size_t)gc * p.taps, p.G * dk + gc, k[e]);
      }
#pragma unroll
      for (uint32_t t = 0; t < kTT; ++t) { qq[t] = fmaf(q[e][t], q[e][t], qq[t]); kk[t] = fmaf(k[e][t], k[e][t], kk[t]); }
    }
#pragma unroll
    for (uint32_t t = 0; t < kTT; ++t) {
      const float rq = p.q_scale / sqrtf(warp_sum(qq[t]) + p.unit_eps), rk = 1.0f / sqrtf(warp_sum(kk[t]) + p.unit_eps);
      const size_t at = ((row0 + t) * p.G + g) * w.dkp;
#pragma unroll
      for (int e = 0; e < CH; ++e) {
        const uint32_t c = lane + 32 * e;
        q[e][t] *= rq; k[e][t] *= rk;
        if (c < w.dkp) { w.q[at + c] = q[e][t]; w.k[at + c] = k[e][t]; }
      }
    }
    float dot_k[6], dot_q[10];  // (t, s) = 10, 20, 21, 30, 31, 32 and 00, 10, 11, 20, 21, 22, 30, 31, 32, 33
    int nk = 0, nq = 0;
#pragma unroll
    for (uint32_t t = 0; t < kTT; ++t)
#pragma unroll
      for (uint32_t s = 0; s <= t; ++s) {
        float a = 0.0f, c = 0.0f;
#pragma unroll
        for (int e = 0; e < CH; ++e) { a = fmaf(k[e][t], k[e][s], a); c = fmaf(q[e][t], k[e][s], c); }
        if (s < t) dot_k[nk++] = warp_sum(a);
        dot_q[nq++] = warp_sum(c);
      }
    for (uint32_t i = lane; i < rep; i += 32) {
      const uint32_t h = g * rep + i;
      float gt[kTT], beta[kTT];
#pragma unroll
      for (uint32_t t = 0; t < kTT; ++t) {
        gt[t] = t < nt ? decay_of(p.a_log[h], p.a[(src0 + t) * p.ld_a + h]) : 1.0f;
        beta[t] = t < nt ? p.beta[(src0 + t) * p.ld_beta + h] : 0.0f;
      }
      BlockNumbers n;
      float G = 1.0f;
      int ia = 0, iq = 0;
      n.A[6] = 0.0f; n.A[7] = 0.0f;
#pragma unroll
      for (uint32_t t = 0; t < kTT; ++t) {
        G *= gt[t];
        n.G[t] = G; n.beta[t] = beta[t]; n.bG[t] = beta[t] * G;
#pragma unroll
        for (uint32_t s = 0; s < kTT; ++s) {
          float D = 1.0f;
#pragma unroll
          for (uint32_t j = 0; j < kTT; ++j)
            if (j > s && j <= t) D *= gt[j];
          if (s < t) n.A[ia++] = beta[t] * D * dot_k[(t * (t - 1)) / 2 + s];
          n.Q[t][s] = s <= t ? D * dot_q[iq++] : 0.0f;
          if (t == kTT - 1) n.D[s] = D;
        }
      }
      float4* dst = reinterpret_cast<float4*>(w.sc) + (((size_t)b * tiles + tile) * p.H + h) * (kNumbers / 4);
      const float4* src = reinterpret_cast<const float4*>(&n);
#pragma unroll
      for (uint32_t e = 0; e < kNumbers / 4; ++e) dst[e] = src[e];
    }
  } else {
    const uint32_t c0 = (unit - p.G) * kValueBlock, c1 = min(p.H * dv, c0 + kValueBlock);
    for (uint32_t c = c0 + lane; c < c1; c += 32) {
      float y[kTT];
      conv(p.v + c, p.ld_v, p.conv_v + (size_t)c * p.taps, 2 * p.G * dk + c, y);
      const uint32_t at = c / dv * w.dvp + c % dv;
#pragma unroll
      for (uint32_t t = 0; t < kTT; ++t) w.v[(row0 + t) * p.H * w.dvp + at] = y[t];
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

// grid (blocks of kOwners * C value columns, heads, sequences); a half warp owns C columns (1 or 2), KPL key channels per
// lane; `tb` blocks of tokens in each of two buffers of [4 tb][2 (q, k)][16 KPL], [4 tb][kOwners * C] values, [tb] numbers.
template <int KPL, int C>
__global__ void __launch_bounds__(kCThreads) delta_scan_kernel(const DeltaParams p, const Work w, uint32_t tb) {
  extern __shared__ __align__(16) float sm[];
  constexpr uint32_t kRow = kLanes * KPL, kCols = kOwners * C;
  constexpr int K2 = KPL / 2;
  constexpr bool kAhead = KPL <= 8;  // the next block's rows are requested before this one's sums are exchanged
  const uint32_t h = blockIdx.y, b = blockIdx.z, dk = p.dk, dv = p.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t l = tid & (kLanes - 1), cl = tid / kLanes * C, cb = blockIdx.x * kCols, T = p.T, g = h / (p.H / p.G), nblocks = w.Tp / kTT;
  const uint32_t buf_floats = tb * (kTT * (2 * kRow + kCols) + kNumbers);
  for (uint32_t i = tid; i < 2 * buf_floats; i += kCThreads) sm[i] = 0.0f;  // channels past dkp stay zero
  __syncthreads();
  grid_dependency_wait();
  grid_launch_dependents();
  auto fetch = [&](uint32_t b0, uint32_t buf) {
    float* base = sm + buf * buf_floats;
    const uint32_t n = min(tb, nblocks - b0) * kTT;
    for (uint32_t t = warp; t < n; t += kCThreads / 32) {
      const size_t row = (size_t)b * w.Tp + b0 * kTT + t;
      const float *q = w.q + (row * p.G + g) * w.dkp, *k = w.k + (row * p.G + g) * w.dkp, *v = w.v + row * p.H * w.dvp + (size_t)h * w.dvp + cb;
      float* d = base + t * 2 * kRow;
      for (uint32_t e = 4 * lane; e < w.dkp; e += 128) {
        cp_async16(d + e, q + e);
        cp_async16(d + kRow + e, k + e);
      }
      if (4 * lane < kCols && cb + 4 * lane < w.dvp) cp_async16(base + tb * kTT * 2 * kRow + t * kCols + 4 * lane, v + 4 * lane);
      if (t % kTT == 0 && lane >= 16 && lane < 16 + kNumbers / 4) {
        const uint32_t e = 4 * (lane - 16);
        cp_async16(base + tb * kTT * (2 * kRow + kCols) + t / kTT * kNumbers + e, w.sc + (((size_t)b * nblocks + b0 + t / kTT) * p.H + h) * kNumbers + e);
      }
    }
    cp_commit();
  };
  fetch(0, 0);
  f32x2 S[C][K2];
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
  // Where the sums over the lanes end up: sum number i = (0: with k, 1: with q; token; column) on the lane whose bits are
  // i's backwards.
  constexpr int N = 8 * C;
  constexpr int kBits = C == 2 ? 4 : 3;
  uint32_t mine = 0;
#pragma unroll
  for (int s = 0; s < kBits; ++s) mine |= (l >> s & 1u) << (kBits - 1 - s);
  const uint32_t mt = mine / C % kTT, mj = mine % C;  // this lane's token and column
  const bool writer = (l & 1) && l < (1u << kBits) && cb + cl + mj < dv;
  uint32_t buf = 0;
  for (uint32_t b0 = 0; b0 < nblocks; b0 += tb, buf ^= 1) {
    if (b0 + tb < nblocks) { fetch(b0 + tb, buf ^ 1); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    const float* s = sm + buf * buf_floats;
    const float *sv = s + tb * kTT * 2 * kRow, *sn = sv + tb * kTT * kCols;
    const uint32_t n = min(tb, nblocks - b0);
    struct Rows { f32x2 x[kTT][K2]; };
    auto load = [&](uint32_t blk, uint32_t which, Rows& r) {  // 0: q, 1: k
#pragma unroll
      for (uint32_t t = 0; t < kTT; ++t)
#pragma unroll
        for (int e = 0; e < KPL / 4; ++e) {
          const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(s + (blk * kTT + t) * 2 * kRow + which * kRow + 4 * (l + kLanes * e));
          r.x[t][2 * e] = v.x; r.x[t][2 * e + 1] = v.y;
        }
    };
    const size_t orow = (size_t)p.H * dv;
    float* out = w.o + ((size_t)b * T + b0 * kTT + mt) * orow + (size_t)h * dv + cb + cl + mj;
    Rows k, q;
    load(0, 1, k);
    load(0, 0, q);
#pragma unroll 2
    for (uint32_t blk = 0; blk < n; ++blk) {
      float z[N];
#pragma unroll
      for (uint32_t t = 0; t < kTT; ++t)
#pragma unroll
        for (int j = 0; j < C; ++j) {
          f32x2 a = mul2(k.x[t][0], S[j][0]), c = mul2(q.x[t][0], S[j][0]);
#pragma unroll
          for (int i = 1; i < K2; ++i) { a = fma2(k.x[t][i], S[j][i], a); c = fma2(q.x[t][i], S[j][i], c); }
          const float2 a2 = unpack2(a), c2 = unpack2(c);
          z[t * C + j] = a2.x + a2.y; z[N / 2 + t * C + j] = c2.x + c2.y;
        }
      Rows nk;
      if (kAhead) { load(min(blk + 1, n - 1), 1, nk); load(min(blk + 1, n - 1), 0, q); }
      const float* num = sn + blk * kNumbers;
      const float4 G = *reinterpret_cast<const float4*>(num), be = *reinterpret_cast<const float4*>(num + 4), bG = *reinterpret_cast<const float4*>(num + 8);
      const float4 A0 = *reinterpret_cast<const float4*>(num + 12), Q = *reinterpret_cast<const float4*>(num + 20 + 4 * mt), D = *reinterpret_cast<const float4*>(num + 36);
      const float2 A1 = *reinterpret_cast<const float2*>(num + 16);
      float v[kTT][C];
#pragma unroll
      for (uint32_t t = 0; t < kTT; ++t) {
        const float* d = sv + (blk * kTT + t) * kCols + cl;
        if constexpr (C == 2) { const float2 x = *reinterpret_cast<const float2*>(d); v[t][0] = x.x; v[t][1] = x.y; }
        else v[t][0] = *d;
      }
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
        } else {
          z[0] += __shfl_xor_sync(0xFFFFFFFFu, z[0], bit);
        }
      }
      float u[kTT][C];
#pragma unroll
      for (uint32_t t = 0; t < kTT; ++t)
#pragma unroll
        for (int j = 0; j < C; ++j) {
          const uint32_t i = t * C + j;  // below N / 2: a sum with k
          uint32_t from = 0;
#pragma unroll
          for (int e = 0; e < kBits; ++e) from |= (i >> e & 1u) << (kBits - 1 - e);
          u[t][j] = __shfl_sync(0xFFFFFFFFu, z[0], from, kLanes);
        }
#pragma unroll
      for (int j = 0; j < C; ++j) {
        u[0][j] = fmaf(be.x, v[0][j], -(bG.x * u[0][j]));
        u[1][j] = fmaf(-A0.x, u[0][j], fmaf(be.y, v[1][j], -(bG.y * u[1][j])));
        u[2][j] = fmaf(-A0.z, u[1][j], fmaf(-A0.y, u[0][j], fmaf(be.z, v[2][j], -(bG.z * u[2][j]))));
        u[3][j] = fmaf(-A1.y, u[2][j], fmaf(-A1.x, u[1][j], fmaf(-A0.w, u[0][j], fmaf(be.w, v[3][j], -(bG.w * u[3][j])))));
      }
      const f32x2 gg = pack2(G.w, G.w);
#pragma unroll
      for (int j = 0; j < C; ++j) {
        const float w0 = D.x * u[0][j], w1 = D.y * u[1][j], w2 = D.z * u[2][j], w3 = u[3][j];
        const f32x2 p0 = pack2(w0, w0), p1 = pack2(w1, w1), p2 = pack2(w2, w2), p3 = pack2(w3, w3);
#pragma unroll
        for (int i = 0; i < K2; ++i)
          S[j][i] = fma2(k.x[3][i], p3, fma2(k.x[2][i], p2, fma2(k.x[1][i], p1, fma2(k.x[0][i], p0, mul2(gg, S[j][i])))));
      }
      {
        float a = mt == 0 ? G.x : mt == 1 ? G.y : mt == 2 ? G.z : G.w;
        a *= z[0];
        a = fmaf(Q.x, C == 2 && mj ? u[0][C - 1] : u[0][0], a);
        a = fmaf(Q.y, C == 2 && mj ? u[1][C - 1] : u[1][0], a);
        a = fmaf(Q.z, C == 2 && mj ? u[2][C - 1] : u[2][0], a);
        a = fmaf(Q.w, C == 2 && mj ? u[3][C - 1] : u[3][0], a);
        if (writer && (b0 + blk) * kTT + mt < T) out[(size_t)blk * kTT * orow] = a;
      }
      if (kAhead) k = nk;
      else if (blk + 1 < n) { load(blk + 1, 1, k); load(blk + 1, 0, q); }
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
  const uint32_t tb = KPL <= 8 ? 8 : 4;
  const size_t smem = 2 * (size_t)tb * (kTT * (2 * kLanes * KPL + kCols) + kNumbers) * sizeof(float);
  return ruai_launch(c, delta_scan_kernel<KPL, C>, dim3((p.dv + kCols - 1) / kCols, p.H, B), dim3(kCThreads), smem, true, p, w, tb);
}
template <int KPL>
cudaError_t columns_scan(ruai_ctx* c, const DeltaParams& p, const Work& w, uint32_t B) {
  // two columns per thread as long as most SMs get a CTA
  const uint64_t ctas = (uint64_t)((p.dv + 2 * kOwners - 1) / (2 * kOwners)) * p.H * B;
  if constexpr (KPL <= 8)
    if (ctas >= (uint64_t)c->sm_count * 3 / 4) return launch_scan<KPL, 2>(c, p, w, B);
  return launch_scan<KPL, 1>(c, p, w, B);
}

template <int N>
cudaError_t launch_conv(ruai_ctx* c, const DeltaParams& p, const Work& w, uint32_t B) {
  const uint32_t units = p.G + (p.H * p.dv + kValueBlock - 1) / kValueBlock, tiles = w.Tp / kTT, items = B * tiles * units;
  const dim3 grid((items + 7) / 8);
  return p.dk <= 128 ? ruai_launch(c, delta_conv_kernel<N, 4>, grid, dim3(256), 0, true, p, w, items, units, tiles)
                     : ruai_launch(c, delta_conv_kernel<N, 8>, grid, dim3(256), 0, true, p, w, items, units, tiles);
}

}  // namespace

size_t ruai_delta_work(const DeltaParams& p, uint32_t rows, uint32_t B) {
  const size_t padded = rows + (size_t)B * (kTT - 1);
  return padded * (2 * (size_t)p.G * up4(p.dk) + (size_t)p.H * up4(p.dv) + (size_t)p.H * kNumbers / kTT + (size_t)p.H * p.dv);
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
  const Work w = work_of(p, B);
  RUAI_CUDA(c, p.taps <= 4 ? launch_conv<4>(c, p, w, B) : launch_conv<kConvMax>(c, p, w, B));
  const uint32_t C = 2 * p.G * p.dk + p.H * p.dv;
  RUAI_CUDA(c, ruai_launch(c, conv_history_kernel, dim3((C + 255) / 256, std::min(p.T, p.taps), B), dim3(256), 0, true, p));
  RUAI_CUDA(c, p.dk <= 64 ? columns_scan<4>(c, p, w, B) : p.dk <= 128 ? columns_scan<8>(c, p, w, B) : columns_scan<16>(c, p, w, B));
  RecurrenceParams r;
  r.o = w.o; r.H = p.H; r.dv = p.dv; r.eps = p.eps; r.norm = p.norm; r.gate = p.gate; r.ld_gate = p.ld_gate;
  r.out = p.out; r.out_ld = p.out_ld; r.out_dtype = p.out_dtype;
  return ruai_head_norm(c, r, rows);
}
