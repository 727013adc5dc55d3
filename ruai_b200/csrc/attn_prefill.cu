// Causal attention over the KV cache for MANY query positions at once (prefill): queries in tiles, so that a cached key
// or value is read from memory once per tile of 16 queries instead of once per query.
//
// Semantics are those of attention_kernel (decode_ops.cu), i.e. of `scaled_dot_product_attention` with the causal
// offset of functional.rs:238-247 / 281-296: query t of the new block sees keys 0 .. past + t.  q is rotated and the
// new keys / values are appended before (rope_kv_kernel).  Everything is f32 on the CUDA cores: softmax(q k^T / sqrt(hd)) v
// with a running maximum and sum per row (the order of the additions differs from the CPU's, as every GPU kernel's does;
// the parity tests bound the difference).
//
// A CTA owns (sequence, KV head, tile of QT queries): rows = QT queries x the REP query heads of the group, 64 rows
// (48 for groups of three).  Eight computing warps own an eighth of the rows each and never need each other after the query tile is in shared memory; a ninth warp's
// first lane streams the keys and values, 64 at a time, through two shared-memory buffers with bulk copies (keys row by
// row into rows padded by four floats, so that a lane per key reads them without bank conflicts).  Per chunk a warp
// computes its rows' scores (a lane per key, two keys per lane, all of the warp's rows at once: a key row is read from
// shared memory once per warp), updates the rows' running softmax, leaves the probabilities in its own rows of a
// shared tile and accumulates probabilities x values (a lane per four elements of the head dimension).
//
// Keys may also lie apart (one head's part per position of a wider row, the last elements in a row shared by the heads):
// the copying warp then puts every key together from two copies.
//
// The same kernel serves windows with kept first positions (chunks nothing of which a tile sees are not read), values of
// another width than the keys, and two score maps per head over the same values (MAPS = 2: half of the warps own the
// rows of each map; the maps meet in shared memory at the end).
#include "common.cuh"
#include "decode_ops.cuh"
#include "pipeline.cuh"

namespace {

using namespace pipe;

constexpr int kKC = 64;        // keys per chunk
constexpr int kWarps = 8;      // computing warps
constexpr int kThreads = (kWarps + 1) * 32;
constexpr size_t kSmemMax = 227 * 1024 - 256;  // what a CTA can have, less the static part

template <int REP, int kQT, int MAPS>
__global__ void __launch_bounds__(kThreads) attention_prefill_kernel(const AttnParams p, uint32_t hd4_per_lane, uint32_t nbuf) {
  constexpr int kMapRows = kQT * REP, kRows = kMapRows * MAPS;  // rows: map, then query, then head
  constexpr int R = kRows / kWarps;     // rows per warp
  static_assert(kRows % kWarps == 0 && kMapRows % R == 0, "rows must share out over the warps, each within one map");
  extern __shared__ __align__(128) unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t full[2], empty[2];
  __shared__ int s_abort;
  const uint32_t hd = p.hd, vd = p.vd, krow = MAPS * hd, kstride = krow + 4u;
  float* qs = reinterpret_cast<float*>(smem_raw);                  // [kRows][hd]
  float* ks = qs + (size_t)kRows * hd;                              // [nbuf][kKC][krow + 4]
  float* vs = ks + nbuf * (size_t)kKC * kstride;                    // [nbuf][kKC][vd]
  float* ps = vs + nbuf * (size_t)kKC * vd;                         // [kRows][kKC]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // the tiles with the most keys first: they are the long ones
  const uint32_t subs = gridDim.z;  // CTAs that share a KV head's query heads, REP each
  const uint32_t bk = blockIdx.y, b = bk / p.KV, kvh = bk % p.KV, q0 = (gridDim.x - 1u - blockIdx.x) * kQT;
  const uint32_t head0 = (kvh * subs + blockIdx.z) * REP;
  if (tid == 0) {
    for (int i = 0; i < 2; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], kWarps); }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    s_abort = 0;
  }
  grid_dependency_wait();
  grid_launch_dependents();
  const uint32_t past = (uint32_t)*p.len;
  const uint32_t nq = min((uint32_t)kQT, p.T - q0);
  uint32_t kmax = past + q0 + nq;  // keys 0 .. kmax - 1 are seen by the tile's last query
  const bool over = kmax > p.cap;  // the device's position is not the host's: touch nothing beyond the cache, tell the host
  if (over) {
    kmax = 0;
    if (tid == 0 && p.status) atomicCAS(p.status, 0, 5);
  }
  // chunks that hold a kept first position, then those from the first query's window on
  const uint32_t all_chunks = (kmax + kKC - 1) / kKC, first = past + q0;
  const uint32_t lo = p.window && first + 1u > p.window ? first + 1u - p.window : 0u;
  const uint32_t kept_chunks = (min(p.keep, kmax) + kKC - 1) / kKC, lo_chunk = min(max(lo / kKC, kept_chunks), all_chunks);
  const uint32_t nchunks = kept_chunks + all_chunks - lo_chunk;
  auto chunk_at = [&](uint32_t i) { return i < kept_chunks ? i : lo_chunk + (i - kept_chunks); };
  // the query tile: row r = map * kMapRows + qi * REP + h
  for (uint32_t i = tid; i < (uint32_t)kRows * (hd / 4); i += kThreads) {
    const uint32_t r = i / (hd / 4), e4 = i % (hd / 4), mp = r / kMapRows, qi = (r % kMapRows) / REP, h = r % REP;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (qi < nq) v = *reinterpret_cast<const float4*>(p.q + (size_t)(b * p.T + q0 + qi) * p.q_ld + (size_t)((head0 + h) * MAPS + mp) * hd + 4 * e4);
    reinterpret_cast<float4*>(qs)[i] = v;
  }
  __syncthreads();
  const bool apart = p.k_pos != 0;
  const float* kbase = p.kcache + (apart ? b * p.k_batch + (size_t)kvh * p.k_head : (size_t)bk * p.cap * krow);
  const float* vbase = p.vcache + (apart ? b * p.v_batch + (size_t)kvh * p.v_head : (size_t)bk * p.cap * vd);

  if (warp == kWarps) {
    // ===== the copying warp =====
    if (apart) {  // many copies: a lane per key
      const float* k2 = p.hd2 ? p.k2 + b * p.k2_batch : nullptr;
      const uint32_t hd1 = krow - p.hd2;
      for (uint32_t c = 0; c < nchunks; ++c) {
        const uint32_t buf = c % nbuf;
        if (__any_sync(0xFFFFFFFFu, c >= nbuf && (s_abort || !mbar_wait(&empty[buf], (c / nbuf - 1u) & 1u)))) { s_abort = 1; break; }
        const uint32_t k0 = chunk_at(c) * kKC, nk = min((uint32_t)kKC, kmax - k0);
        if (lane == 0) mbar_expect_tx(&full[buf], nk * (krow + vd) * 4u);
        __syncwarp();
        for (uint32_t k = lane; k < nk; k += 32) {
          float* dst = ks + ((size_t)buf * kKC + k) * kstride;
          bulk_load(dst, kbase + (size_t)(k0 + k) * p.k_pos, hd1 * 4u, &full[buf]);
          if (k2) bulk_load(dst + hd1, k2 + (size_t)(k0 + k) * p.k2_pos, p.hd2 * 4u, &full[buf]);
          bulk_load(vs + ((size_t)buf * kKC + k) * vd, vbase + (size_t)(k0 + k) * p.v_pos, vd * 4u, &full[buf]);
        }
      }
    } else if (lane == 0) {
      for (uint32_t c = 0; c < nchunks; ++c) {
        const uint32_t buf = c % nbuf;
        if (c >= nbuf && (s_abort || !mbar_wait(&empty[buf], (c / nbuf - 1u) & 1u))) { s_abort = 1; break; }
        const uint32_t k0 = chunk_at(c) * kKC, nk = min((uint32_t)kKC, kmax - k0), row = krow * 4u;
        mbar_expect_tx(&full[buf], nk * (row + vd * 4u));
        for (uint32_t k = 0; k < nk; ++k) bulk_load(ks + ((size_t)buf * kKC + k) * kstride, kbase + (size_t)(k0 + k) * krow, row, &full[buf]);
        bulk_load(vs + (size_t)buf * kKC * vd, vbase + (size_t)k0 * vd, nk * vd * 4u, &full[buf]);
      }
    }
    return;
  }

  // ===== computing warps =====
  const uint32_t row0 = (uint32_t)warp * R, map = row0 / kMapRows, mrow0 = row0 % kMapRows;
  float m_run[R], l_run[R];
  float4 o[R][2];  // this lane's elements 4 (lane + 32 j) .. of the head dimension, j < hd4_per_lane <= 2
#pragma unroll
  for (int r = 0; r < R; ++r) {
    m_run[r] = p.sink ? p.sink[head0 + (mrow0 + r) % REP] : -INFINITY;  // a sink is a first term without a value
    l_run[r] = p.sink ? 1.0f : 0.0f;
    o[r][0] = make_float4(0.f, 0.f, 0.f, 0.f); o[r][1] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (uint32_t c = 0; c < nchunks; ++c) {
    const uint32_t buf = c % nbuf, k0 = chunk_at(c) * kKC, nk = min((uint32_t)kKC, kmax - k0);
    if (s_abort || !mbar_wait(&full[buf], (c / nbuf) & 1u)) { s_abort = 1; break; }
    const float* kb = ks + (size_t)buf * kKC * kstride + map * hd;
    const float* vb = vs + (size_t)buf * kKC * vd;
    // ---- scores: this lane's keys `lane` and `lane + 32` against the warp's R rows ----
    float s0[R], s1[R];
#pragma unroll
    for (int r = 0; r < R; ++r) { s0[r] = 0.0f; s1[r] = 0.0f; }
    const float4* k0p = reinterpret_cast<const float4*>(kb + (size_t)lane * kstride);
    const float4* k1p = reinterpret_cast<const float4*>(kb + (size_t)(lane + 32) * kstride);
    const float4* qp = reinterpret_cast<const float4*>(qs + (size_t)row0 * hd);
    for (uint32_t e4 = 0; e4 < hd / 4; ++e4) {
      const float4 a = k0p[e4], bq = k1p[e4];
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const float4 qv = qp[(size_t)r * (hd / 4) + e4];
        s0[r] = fmaf(qv.x, a.x, s0[r]); s0[r] = fmaf(qv.y, a.y, s0[r]); s0[r] = fmaf(qv.z, a.z, s0[r]); s0[r] = fmaf(qv.w, a.w, s0[r]);
        s1[r] = fmaf(qv.x, bq.x, s1[r]); s1[r] = fmaf(qv.y, bq.y, s1[r]); s1[r] = fmaf(qv.z, bq.z, s1[r]); s1[r] = fmaf(qv.w, bq.w, s1[r]);
      }
    }
    // ---- running softmax per row; probabilities into the warp's rows of the shared tile ----
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const uint32_t qpos = past + q0 + (mrow0 + r) / REP;  // the last key this row's query sees
      const uint32_t qlo = p.window && qpos + 1u > p.window ? qpos + 1u - p.window : 0u;  // the first but for the kept ones
      const uint32_t key0 = k0 + lane, key1 = key0 + 32u;
      float a = (key0 <= qpos && (key0 >= qlo || key0 < p.keep) && (uint32_t)lane < nk) ? s0[r] * p.scale : -INFINITY;
      float bq = (key1 <= qpos && (key1 >= qlo || key1 < p.keep) && (uint32_t)lane + 32u < nk) ? s1[r] * p.scale : -INFINITY;
      float mx = fmaxf(a, bq);
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, off));
      const float m_new = fmaxf(m_run[r], mx);
      const float p0 = a == -INFINITY ? 0.0f : expf(a - m_new), p1 = bq == -INFINITY ? 0.0f : expf(bq - m_new);
      float sum = p0 + p1;
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xFFFFFFFFu, sum, off);
      const float corr = m_run[r] == -INFINITY ? 0.0f : expf(m_run[r] - m_new);
      l_run[r] = fmaf(l_run[r], corr, sum);
      m_run[r] = m_new;
      o[r][0].x *= corr; o[r][0].y *= corr; o[r][0].z *= corr; o[r][0].w *= corr;
      o[r][1].x *= corr; o[r][1].y *= corr; o[r][1].z *= corr; o[r][1].w *= corr;
      ps[(size_t)(row0 + r) * kKC + lane] = p0;
      ps[(size_t)(row0 + r) * kKC + lane + 32] = p1;
    }
    __syncwarp();
    // ---- values: o[r] += sum_k p[r][k] v[k], four keys at a time (keys past nk carry probability 0) ----
    const uint32_t nk4 = (nk + 3u) & ~3u;
    for (uint32_t k = 0; k < nk4; k += 4) {
      float4 pr[R];
#pragma unroll
      for (int r = 0; r < R; ++r) pr[r] = *reinterpret_cast<const float4*>(ps + (size_t)(row0 + r) * kKC + k);
#pragma unroll
      for (uint32_t j = 0; j < 2; ++j) {
        if (j < hd4_per_lane) {
          const uint32_t e4 = lane + 32u * j;
          if (e4 < vd / 4) {
            const float4 v0 = reinterpret_cast<const float4*>(vb + (size_t)(k + 0) * vd)[e4];
            const float4 v1 = k + 1 < nk ? reinterpret_cast<const float4*>(vb + (size_t)(k + 1) * vd)[e4] : make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 v2 = k + 2 < nk ? reinterpret_cast<const float4*>(vb + (size_t)(k + 2) * vd)[e4] : make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 v3 = k + 3 < nk ? reinterpret_cast<const float4*>(vb + (size_t)(k + 3) * vd)[e4] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int r = 0; r < R; ++r) {
              o[r][j].x = fmaf(pr[r].x, v0.x, o[r][j].x); o[r][j].y = fmaf(pr[r].x, v0.y, o[r][j].y); o[r][j].z = fmaf(pr[r].x, v0.z, o[r][j].z); o[r][j].w = fmaf(pr[r].x, v0.w, o[r][j].w);
              o[r][j].x = fmaf(pr[r].y, v1.x, o[r][j].x); o[r][j].y = fmaf(pr[r].y, v1.y, o[r][j].y); o[r][j].z = fmaf(pr[r].y, v1.z, o[r][j].z); o[r][j].w = fmaf(pr[r].y, v1.w, o[r][j].w);
              o[r][j].x = fmaf(pr[r].z, v2.x, o[r][j].x); o[r][j].y = fmaf(pr[r].z, v2.y, o[r][j].y); o[r][j].z = fmaf(pr[r].z, v2.z, o[r][j].z); o[r][j].w = fmaf(pr[r].z, v2.w, o[r][j].w);
              o[r][j].x = fmaf(pr[r].w, v3.x, o[r][j].x); o[r][j].y = fmaf(pr[r].w, v3.y, o[r][j].y); o[r][j].z = fmaf(pr[r].w, v3.z, o[r][j].z); o[r][j].w = fmaf(pr[r].w, v3.w, o[r][j].w);
            }
          }
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[buf]);  // this warp is done with the chunk's keys and values
  }
  // ---- out = o / l; two maps: the second's rows go through shared memory (the chunk buffers, no longer needed) ----
  float* other = ks;  // [kMapRows][vd]
  if constexpr (MAPS == 2) {
    asm volatile("bar.sync 1, 256;" ::: "memory");  // the computing warps: everyone is through with the last chunk
    if (map == 1) {
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const float inv = 1.0f / l_run[r];
#pragma unroll
        for (uint32_t j = 0; j < 2; ++j) {
          const uint32_t e4 = lane + 32u * j;
          if (j < hd4_per_lane && e4 < vd / 4)
            reinterpret_cast<float4*>(other + (size_t)(mrow0 + r) * vd)[e4] = make_float4(o[r][j].x * inv, o[r][j].y * inv, o[r][j].z * inv, o[r][j].w * inv);
        }
      }
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
  }
  if (s_abort) {  // only here: every computing warp has to come to both barriers
    if (lane == 0 && p.status) atomicCAS(p.status, 0, 3);
    return;
  }
  if (MAPS == 2 && map == 1) return;
  const float lam = MAPS == 2 ? *p.lambda : 0.0f;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const uint32_t row = mrow0 + r, qi = row / REP, h = row % REP;
    if (qi >= nq || over) continue;
    const float inv = (p.gate ? p.gate[(size_t)(b * p.T + q0 + qi) * p.ld_gate + head0 + h] : 1.0f) / l_run[r];
    const size_t at = (size_t)(b * p.T + q0 + qi) * p.out_ld + (size_t)(head0 + h) * p.vd_out;
    float4 y[2];
    float ss = 0.0f;
#pragma unroll
    for (uint32_t j = 0; j < 2; ++j) {
      const uint32_t e4 = lane + 32u * j;
      y[j] = make_float4(o[r][j].x * inv, o[r][j].y * inv, o[r][j].z * inv, o[r][j].w * inv);
      if (MAPS == 2 && j < hd4_per_lane && e4 < vd / 4) {
        const float4 z = reinterpret_cast<const float4*>(other + (size_t)row * vd)[e4];
        y[j].x -= lam * z.x; y[j].y -= lam * z.y; y[j].z -= lam * z.z; y[j].w -= lam * z.w;  // columns past vd_out are zero in both maps
        ss = fmaf(y[j].x, y[j].x, ss); ss = fmaf(y[j].y, y[j].y, ss); ss = fmaf(y[j].z, y[j].z, ss); ss = fmaf(y[j].w, y[j].w, ss);
      }
    }
    float f = 1.0f;
    if constexpr (MAPS == 2) {
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, off);
      f = p.out_scale / sqrtf(ss / (float)p.vd_out + p.eps);
    }
#pragma unroll
    for (uint32_t j = 0; j < 2; ++j) {
      const uint32_t e4 = lane + 32u * j;
      if (j < hd4_per_lane && e4 < vd / 4) {
        const float v[4] = {y[j].x * f, y[j].y * f, y[j].z * f, y[j].w * f};
        if (p.out_dtype == RUAI_F32 && p.vd_out % 4 == 0 && p.out_ld % 4 == 0) reinterpret_cast<float4*>(p.out + at)[e4] = make_float4(v[0], v[1], v[2], v[3]);
        else {
#pragma unroll
          for (uint32_t i = 0; i < 4; ++i)
            if (4 * e4 + i < p.vd_out) store_from_f32(p.out, p.out_dtype, at + 4 * e4 + i, v[i]);
        }
      }
    }
  }
}

template <int REP, int kQT, int MAPS>
cudaError_t launch(ruai_ctx* c, const AttnParams& p, uint32_t B, uint32_t subs, size_t smem, uint32_t hd4_per_lane, uint32_t nbuf) {
  static bool done[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(attention_prefill_kernel<REP, kQT, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax);
    if (e != cudaSuccess) return e;
    done[dev & 63] = true;
  }
  const dim3 grid((p.T + kQT - 1) / kQT, B * p.KV, subs);
  return ruai_launch(c, attention_prefill_kernel<REP, kQT, MAPS>, grid, dim3(kThreads), smem, true, p, hd4_per_lane, nbuf);
}

constexpr int tile_queries(int rep, int maps = 1) { return (rep == 3 ? 16 : 64 / rep) / maps; }
size_t smem_bytes(size_t rows, uint32_t maps, uint32_t hd, uint32_t vd, uint32_t nbuf) {
  return (rows * hd + nbuf * (size_t)kKC * (maps * hd + 4) + nbuf * (size_t)kKC * vd + rows * kKC) * sizeof(float);
}
bool widths_fit(uint32_t hd, uint32_t vd) { return hd % 4 == 0 && hd <= 256 && vd % 4 == 0 && vd <= 256; }

}  // namespace

bool ruai_attention_prefill_fits(uint32_t hd, uint32_t vd) { return widths_fit(hd, vd) && smem_bytes(tile_queries(1), 1, hd, vd, 1) <= kSmemMax; }

// 1: launched; 0: this shape is not taken (the caller uses the kernel for few queries); < 0: error.
int ruai_attention_prefill(ruai_ctx* c, const AttnParams& p_in, uint32_t B, uint32_t rep_in) {
  AttnParams p = p_in;
  if (p.maps == 0) p.maps = 1;
  if (p.vd == 0) p.vd = p.hd;
  if (p.vd_out == 0) p.vd_out = p.vd;
  if (p.fuse || p.T < 8 || !widths_fit(p.hd, p.vd) || p.maps > 2 || (p.k_pos && p.maps != 1)) return 0;
  // query heads per CTA; other counts are shared out over several CTAs
  uint32_t rep = 1;
  for (uint32_t r : {8u, 4u, 3u, 2u})
    if (rep_in % r == 0) { rep = r; break; }
  const uint32_t subs = rep_in / rep;
  if (subs > 65535 || B * p.KV > 65535) return 0;
  const size_t rows = (size_t)tile_queries((int)rep, (int)p.maps) * rep * p.maps;
  const uint32_t nbuf = smem_bytes(rows, p.maps, p.hd, p.vd, 2) <= kSmemMax ? 2 : 1;
  const size_t smem = smem_bytes(rows, p.maps, p.hd, p.vd, nbuf);
  if (smem > kSmemMax) return 0;
  const uint32_t hd4_per_lane = (p.vd / 4 + 31) / 32;
  cudaError_t e;
  if (p.maps == 1) switch (rep) {
    case 1: e = launch<1, tile_queries(1), 1>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
    case 2: e = launch<2, tile_queries(2), 1>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
    case 3: e = launch<3, tile_queries(3), 1>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
    case 4: e = launch<4, tile_queries(4), 1>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
    default: e = launch<8, tile_queries(8), 1>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
  } else switch (rep) {
    case 1: e = launch<1, tile_queries(1, 2), 2>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
    case 2: e = launch<2, tile_queries(2, 2), 2>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
    case 3: e = launch<3, tile_queries(3, 2), 2>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
    case 4: e = launch<4, tile_queries(4, 2), 2>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
    default: e = launch<8, tile_queries(8, 2), 2>(c, p, B, subs, smem, hd4_per_lane, nbuf); break;
  }
  if (e != cudaSuccess) { ruai_fail(c, RUAI_ERR_CUDA, "prefill attention launch: %s", cudaGetErrorString(e)); return -1; }
  return 1;
}
