// Unquantized Linears: y = x @ W^T for weights kept in bf16 or f32, one row of k elements per output (QL_DENSE).
//
// A launch takes a GROUP of up to eight Linears with the same number of rows, so that the projections of a layer that
// read different inputs (a token-shifted one, five interpolated ones, the unshifted one of the feed-forward) are still
// one kernel.  Each member has its own epilogue: bias, activation (also of gate / up pairs in neighbouring columns),
// residual, output type, greedy pick.  A member's weight may hold several Linears of one shape, chosen by the output column
// (every head its own) or by the row (every expert its own tokens).
//
//   up to 16 rows  dense_gemv_kernel: the weight streams once through registers (16 bytes per lane and row of W, R rows
//                  of W at a time, the next step's loads in flight; the first ones ahead of the dependency wait), f32
//                  multiply-adds, k shared out over the warps of a CTA where it is long.
//   more, bf16     dense_gemm_kernel: tcgen05 kind::f16.  Weights are the M = 128 operand, rows of x the N operand; both
//                  arrive by TMA with the 128-byte swizzle in a ring of shared-memory stages, the accumulator lives in
//                  tensor memory and is read back a lane per output column, so that stores are coalesced.
//   more, else     dense_simt_kernel: f32 multiply-adds on 64 x 64 tiles (f32 weights: no reduced-precision mode).
// Products and sums are f32 everywhere; bf16 weights and activations enter exactly.  Every mbarrier wait is bounded.
#include <cuda.h>

#include "common.cuh"
#include "gemv_epilogue.cuh"
#include "pipeline.cuh"

namespace dense {

using namespace pipe;

struct Seg {
  const void* w;
  const void* x;
  void* out;
  const float* bias;
  const float* aux;
  const float* resid;
  uint32_t n, k, ldw, ldx, ldo, tile0;
  int act, out_dtype, x_vec;
  // blocks of the weight's rows: see DenseCall
  uint32_t tiles, nb, xblk, oblk, xdiv, wrow0, xcol0;  // tiles of one block's columns; wrow0, xcol0: filled in by pick_seg
  const int32_t* table;
  int table_early;
};
struct Group {
  Seg seg[kDenseGroupMax];
  int nseg;
  uint32_t m;
  int x_dtype;
  // greedy pick of the only member
  int32_t* arg_out;
  unsigned long long* arg_slots;
  int32_t* len_ptr;
  int32_t len_add;
  int* status;
};

__device__ __forceinline__ float gelu_tanh(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__host__ __device__ __forceinline__ bool is_pair(int act) { return act == ACT_SWIGLU || act == ACT_GEGLU || act == ACT_REGLU; }
__device__ __forceinline__ float unary(int act, const float* aux, uint32_t j, float v) {
  switch (act) {
    case ACT_GELU: return gelu_ref(v);
    case ACT_SILU: return v * sigmoid(v);
    case ACT_TANH: return tanhf(v);
    case ACT_SIGMOID: return sigmoid(v);
    case ACT_DECAY: return expf(-expf(v));
    case ACT_FORGET: { const float l = aux[j]; return l + (1.0f - l) * sigmoid(v); }
    default: return v;
  }
}
template <int ACT>
__device__ __forceinline__ float act_of(float l, float v) {
  if constexpr (ACT == ACT_GELU) return gelu_ref(v);
  if constexpr (ACT == ACT_SILU) return v * sigmoid(v);
  if constexpr (ACT == ACT_TANH) return tanhf(v);
  if constexpr (ACT == ACT_SIGMOID) return sigmoid(v);
  if constexpr (ACT == ACT_DECAY) return expf(-expf(v));
  if constexpr (ACT == ACT_FORGET) return l + (1.0f - l) * sigmoid(v);
  return v;
}
__device__ __forceinline__ float pair_act(int act, float gate, float up) {
  return (act == ACT_GEGLU ? gelu_tanh(gate) : act == ACT_REGLU ? fmaxf(gate, 0.0f) : silu_ref(gate)) * up;
}
// Bias, activation, residual and store of column j of one row; pair activations: of the pair (j, j + 1) with sums v, v2.
__device__ __forceinline__ float finish(const Seg& s, uint32_t row, uint32_t j, float v, float v2) {
  if (s.bias) { v += s.bias[j]; if (is_pair(s.act)) v2 += s.bias[j + 1]; }
  size_t o;
  if (is_pair(s.act)) {
    v = pair_act(s.act, v, v2);
    o = (size_t)row * s.ldo + (j >> 1);
  } else {
    v = unary(s.act, s.aux, j, v);
    o = (size_t)row * s.ldo + j;
  }
  if (s.resid) v += s.resid[o];
  store_from_f32(s.out, s.out_dtype, o, v);
  return v;
}
// The same for 32 consecutive rows of one column at once: the column's constants and the residual's values are requested
// before the first store (the compiler cannot move loads over stores).  A lane per column; the warp stays converged.
template <int ACT>
__device__ __forceinline__ void finish_rows(const Seg& s, uint32_t row0, uint32_t m, uint32_t j, float (&v)[32]) {
  constexpr bool kPair = ACT == ACT_GEGLU;  // stands for every pair activation
  const bool in = j < s.n && !(kPair && (j & 1u));
  const uint32_t jj = min(j, s.n - 1);
  const float bias = s.bias ? s.bias[jj] : 0.0f, aux = ACT == ACT_FORGET ? s.aux[jj] : 0.0f;
  const uint32_t nr = min(32u, m - row0);
  const size_t o = (size_t)row0 * s.ldo + (kPair ? j >> 1 : j);
#pragma unroll
  for (int t = 0; t < 32; ++t) {
    v[t] += bias;
    if constexpr (kPair) v[t] = pair_act(s.act, v[t], __shfl_xor_sync(0xFFFFFFFFu, v[t], 1));
    else v[t] = act_of<ACT>(aux, v[t]);
  }
  if (!in) return;
  if (s.resid) {
    float r[32];
#pragma unroll
    for (int t = 0; t < 32; ++t) r[t] = (uint32_t)t < nr ? s.resid[o + (size_t)t * s.ldo] : 0.0f;
#pragma unroll
    for (int t = 0; t < 32; ++t) v[t] += r[t];
  }
  if (s.out_dtype == RUAI_F32) {
    float* p = (float*)s.out + o;
#pragma unroll
    for (int t = 0; t < 32; ++t)
      if ((uint32_t)t < nr) p[(size_t)t * s.ldo] = v[t];
  } else {
#pragma unroll
    for (int t = 0; t < 32; ++t)
      if ((uint32_t)t < nr) store_from_f32(s.out, s.out_dtype, o + (size_t)t * s.ldo, v[t]);
  }
}
// The member that tile `t` of the launch belongs to, copied to shared memory by one thread (static indexing of the
// parameter block: nothing takes its address).
__device__ __forceinline__ void pick_seg(const Group& g, uint32_t t, Seg* dst) {
#pragma unroll
  for (int i = 0; i < kDenseGroupMax; ++i) {
    if (i < g.nseg && t >= g.seg[i].tile0 && (i + 1 >= g.nseg || t < g.seg[(i + 1) % kDenseGroupMax].tile0)) *dst = g.seg[i];
  }
}
// The member's block of tile `t` (its weights, and where its inputs and outputs begin); afterwards s.tile0 is the tile of the
// block's first column.  False: the row tile has no block.  One thread; `row_tile`: the tile of rows.
__device__ __forceinline__ bool pick_block(Seg* s, uint32_t t, uint32_t row_tile, uint32_t w_bytes, uint32_t x_bytes) {
  s->wrow0 = 0; s->xcol0 = 0;
  if (s->nb == 0) return true;
  uint32_t b;
  if (s->table) {
    const int32_t e = __ldcg(s->table + row_tile);
    if (e < 0) return false;
    b = (uint32_t)e;
    s->oblk = 0;
  } else {
    b = (t - s->tile0) / s->tiles;
    s->tile0 += b * s->tiles;
    s->xcol0 = b * s->xblk;
  }
  s->wrow0 = b * s->nb;
  s->w = (const char*)s->w + (size_t)s->wrow0 * s->ldw * w_bytes;
  s->x = (const char*)s->x + (size_t)s->xcol0 * x_bytes;
  s->out = (char*)s->out + (size_t)b * s->oblk * (s->out_dtype == RUAI_F32 ? 4 : 2);
  return true;
}

// ---- few rows -------------------------------------------------------------------------------------

constexpr int kVThreads = 256, kVWarps = kVThreads / 32;

template <typename WT> struct W8;
template <> struct W8<__nv_bfloat16> {
  uint4 a;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { a = ldg_stream_u4(reinterpret_cast<const uint4*>(p)); }
  __device__ __forceinline__ void zero() { a = make_uint4(0, 0, 0, 0); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    const uint32_t u[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(u[i] << 16); f[2 * i + 1] = __uint_as_float(u[i] & 0xFFFF0000u); }
  }
};
template <> struct W8<float> {
  uint4 a, b;
  __device__ __forceinline__ void load(const float* p) {
    a = ldg_stream_u4(reinterpret_cast<const uint4*>(p));
    b = ldg_stream_u4(reinterpret_cast<const uint4*>(p) + 1);
  }
  __device__ __forceinline__ void zero() { a = b = make_uint4(0, 0, 0, 0); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    const uint32_t u[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(u[i]);
  }
};
// Eight elements of a row of x from element kk on; elements past k read as 0.
__device__ __forceinline__ void load_x8(const __nv_bfloat16* x, uint32_t kk, uint32_t k, bool vec, float (&f)[8]) {
  if (vec && kk + 8 <= k) {
    const uint4 a = *reinterpret_cast<const uint4*>(x + kk);
    const uint32_t u[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(u[i] << 16); f[2 * i + 1] = __uint_as_float(u[i] & 0xFFFF0000u); }
  } else {
#pragma unroll
    for (uint32_t i = 0; i < 8; ++i) f[i] = kk + i < k ? __bfloat162float(x[kk + i]) : 0.0f;
  }
}
__device__ __forceinline__ void load_x8(const float* x, uint32_t kk, uint32_t k, bool vec, float (&f)[8]) {
  if (vec && kk + 8 <= k) {
    const float4 a = *reinterpret_cast<const float4*>(x + kk), b = *reinterpret_cast<const float4*>(x + kk + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  } else {
#pragma unroll
    for (uint32_t i = 0; i < 8; ++i) f[i] = kk + i < k ? x[kk + i] : 0.0f;
  }
}

// kw warps share the k of R rows of W; kVWarps / kw such row groups per CTA.  grid (tiles of all members, row tiles of x).
template <typename WT, typename XT, int MT, int R>
__global__ void __launch_bounds__(kVThreads, 2) dense_gemv_kernel(const Group g, uint32_t kw) {
  __shared__ float red[kVWarps][R * MT];
  __shared__ Seg s_seg;
  __shared__ unsigned long long s_best[MT];
  __shared__ bool s_any;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid == 0) {
    pick_seg(g, blockIdx.x, &s_seg);
    if (s_seg.table && !s_seg.table_early) grid_dependency_wait();
    s_any = pick_block(&s_seg, blockIdx.x, blockIdx.y, sizeof(WT), sizeof(XT));
  }
  if (tid < MT) s_best[tid] = 0;
  __syncthreads();
  if (!s_any) {
    grid_dependency_wait();
    return;
  }
  const uint32_t xdiv = s_seg.xdiv;  // above 1 with MT == 1 only
  const uint32_t groups = kVWarps / kw, wk = warp % kw, wr = warp / kw, k = s_seg.k, n = s_seg.n;
  const uint32_t j0 = (blockIdx.x - s_seg.tile0) * groups * R, m0 = blockIdx.y * MT;
  const WT* wp[R];
#pragma unroll
  for (int r = 0; r < R; ++r) wp[r] = reinterpret_cast<const WT*>(s_seg.w) + (size_t)min(j0 + wr * R + r, n - 1) * s_seg.ldw;
  uint32_t kk = (wk * 32 + lane) * 8;
  const uint32_t step = kw * 256;
  W8<WT> cur[R];
  const bool any = j0 + wr * R < n;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    if (any && kk < k) cur[r].load(wp[r] + kk);
    else cur[r].zero();
  }
  grid_dependency_wait();
  grid_launch_dependents();
  float acc[R][MT];
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int i = 0; i < MT; ++i) acc[r][i] = 0.0f;
  const bool vec = s_seg.x_vec != 0;
  const XT* xb = reinterpret_cast<const XT*>(s_seg.x);
  for (; any && kk < k; kk += step) {
    W8<WT> nxt[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      if (kk + step < k) nxt[r].load(wp[r] + kk + step);
      else nxt[r].zero();
    }
    if constexpr (MT <= 2) {  // x of all rows in registers, one row of W expanded at a time
      float xv[MT][8];
#pragma unroll
      for (int i = 0; i < MT; ++i) load_x8(xb + (size_t)(min(m0 + i, g.m - 1) / xdiv) * s_seg.ldx, kk, k, vec, xv[i]);
#pragma unroll
      for (int r = 0; r < R; ++r) {
        float wf[8];
        cur[r].get(wf);
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[r][i] = fmaf(wf[e], xv[i][e], acc[r][i]);
      }
    } else {  // W expanded once, x one row at a time
      float wf[R][8];
#pragma unroll
      for (int r = 0; r < R; ++r) cur[r].get(wf[r]);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        if (m0 + i < g.m) {
          float xv[8];
          load_x8(xb + (size_t)(m0 + i) * s_seg.ldx, kk, k, vec, xv);
#pragma unroll
          for (int r = 0; r < R; ++r)
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[r][i] = fmaf(wf[r][e], xv[e], acc[r][i]);
        }
      }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) cur[r] = nxt[r];
  }
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      float v = acc[r][i];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
      if (lane == ((r * MT + i) & 31)) red[warp][r * MT + i] = v;
    }
  __syncthreads();
  const uint32_t cols = groups * R;
  const bool pair = is_pair(s_seg.act);
  for (uint32_t t = tid; t < cols * MT; t += kVThreads) {
    const uint32_t i = t / cols, c = t % cols, j = j0 + c, row = m0 + i;
    if (row >= g.m || j >= n || (pair && (c & 1u))) continue;
    float v = 0.0f, v2 = 0.0f;
    for (uint32_t q = 0; q < kw; ++q) v += red[(c / R) * kw + q][(c % R) * MT + i];
    if (pair) for (uint32_t q = 0; q < kw; ++q) v2 += red[(c / R) * kw + q][(c % R + 1) * MT + i];
    v = finish(s_seg, row, j, v, v2);
    if (g.arg_out) {
      const uint32_t key = (uint32_t)ordered_bits(v) ^ 0x80000000u;  // ascending with the value; among equal values the larger column
      atomicMax(&s_best[i], ((unsigned long long)key << 32) | j);
    }
  }
  if (!g.arg_out) return;
  __syncthreads();
  // nobody waits for this: dense_pick_kernel reads the slots
  if (tid < MT && m0 + tid < g.m) atomicMax(&g.arg_slots[(size_t)(m0 + tid) * kDenseArgSlots + blockIdx.x % kDenseArgSlots], s_best[tid]);
}

// The rows' picks from the slots the CTAs left, a warp per row; the slots are zero again afterwards.
__global__ void __launch_bounds__(kVThreads) dense_pick_kernel(const Group g) {
  grid_dependency_wait();
  grid_launch_dependents();
  const uint32_t lane = threadIdx.x & 31;
  for (uint32_t row = threadIdx.x >> 5; row < g.m; row += kVWarps) {
    unsigned long long b = 0;
#pragma unroll
    for (uint32_t t = lane; t < kDenseArgSlots; t += 32) {
      unsigned long long* sl = &g.arg_slots[(size_t)row * kDenseArgSlots + t];
      const unsigned long long v = __ldcg(sl);
      *sl = 0;
      b = v > b ? v : b;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const unsigned long long v = __shfl_xor_sync(0xFFFFFFFFu, b, o);
      b = v > b ? v : b;
    }
    if (lane == 0) g.arg_out[row] = (int32_t)(uint32_t)b;
  }
  if (threadIdx.x == 0 && g.len_ptr) *g.len_ptr += g.len_add;
}

// ---- many rows, bf16 --------------------------------------------------------------------------------

constexpr int kTileN = 128;   // columns of the output (rows of W) per CTA: the M of the MMA, the lanes of tensor memory
constexpr int kTileK = 64;    // one 128-byte swizzle row of bf16
constexpr int kGThreads = 192;  // TMA warp, MMA warp, four epilogue warps

struct alignas(64) Maps { CUtensorMap w[kDenseGroupMax], x[kDenseGroupMax]; };

constexpr int stages_of(int nt) { return nt == 128 ? 3 : 4; }
constexpr size_t stage_bytes(int nt) { return (size_t)(kTileN + nt) * kTileK * 2; }
constexpr size_t gemm_smem(int nt) { return stages_of(nt) * stage_bytes(nt) + 1024; }

// Operand descriptor: K-major, 128-byte swizzle, rows of 128 bytes, 1024 bytes between 8-row blocks.
__device__ __forceinline__ uint64_t desc_sw128(uint32_t addr) {
  return (uint64_t)((addr >> 4) & 0x3FFFu) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void tma_2d(void* dst, const CUtensorMap* map, int x, int y, uint64_t* bar) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(smem_u32(dst)),
               "l"((uint64_t)map), "r"(x), "r"(y), "r"(smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ void mma_bf16(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
  asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\ttcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(d), "l"(a), "l"(b),
               "r"(idesc), "r"(accumulate)
               : "memory");
}
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, float (&v)[32]) {
  uint32_t r[32];
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, %17, %18, %19, %20, %21, "
      "%22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
        "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]),
        "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
#pragma unroll
  for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(r[i]);
}

// grid (blocks of NT rows of x, column tiles of all members): the CTAs that run together share few tiles of the weight, which
// so comes from HBM once; all of x stays in the L2.
template <int NT>
__global__ void __launch_bounds__(kGThreads) dense_gemm_kernel(const __grid_constant__ Maps maps, const Group g) {
  constexpr int S = stages_of(NT);
  constexpr uint32_t kABytes = kTileN * kTileK * 2, kBBytes = NT * kTileK * 2;
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t full[S], empty[S], done;
  __shared__ uint32_t s_tmem;
  __shared__ volatile int s_abort;
  __shared__ Seg s_seg;
  __shared__ int s_idx;
  __shared__ bool s_any;
  unsigned char* ring = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);  // the swizzle pattern repeats every 1024 bytes
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid == 0) {
    pick_seg(g, blockIdx.y, &s_seg);
    int idx = 0;
#pragma unroll
    for (int i = 1; i < kDenseGroupMax; ++i)
      if (i < g.nseg && blockIdx.y >= g.seg[i].tile0) idx = i;
    s_idx = idx;
    if (s_seg.table && !s_seg.table_early) grid_dependency_wait();
    s_any = pick_block(&s_seg, blockIdx.y, blockIdx.x, 2, 2);
    for (int s = 0; s < S; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    mbar_init(&done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    s_abort = 0;
  }
  if (g.seg[0].table) {  // a row tile without a block: nothing is allocated or in flight yet
    __syncthreads();
    if (!s_any) {
      grid_dependency_wait();
      return;
    }
  }
  __syncwarp();
  if (warp == 1) tmem_alloc(&s_tmem, NT);
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = s_tmem, k = s_seg.k, nk = (k + kTileK - 1) / kTileK;
  const uint32_t j0 = (blockIdx.y - s_seg.tile0) * kTileN, row0 = blockIdx.x * NT;
  const int wy = (int)(s_seg.wrow0 + j0), xc = (int)s_seg.xcol0;
  if (warp == 0) {
    if (lane == 0) {
      const CUtensorMap* mw = &maps.w[s_idx];
      const CUtensorMap* mx = &maps.x[s_idx];
      const uint32_t pre = min(nk, (uint32_t)S);
      for (uint32_t i = 0; i < pre; ++i) {  // the weights do not depend on the predecessor kernel
        mbar_expect_tx(&full[i], kABytes + kBBytes);
        tma_2d(ring + i * (kABytes + kBBytes), mw, (int)(i * kTileK), wy, &full[i]);
      }
      grid_dependency_wait();
      grid_launch_dependents();
      for (uint32_t i = 0; i < pre; ++i) tma_2d(ring + i * (kABytes + kBBytes) + kABytes, mx, xc + (int)(i * kTileK), (int)row0, &full[i]);
      uint32_t issued = pre;
      for (uint32_t i = pre; i < nk; ++i) {
        const uint32_t s = i % S;
        if (s_abort || !mbar_wait(&empty[s], ((i / S) - 1) & 1u)) { s_abort = 1; break; }
        mbar_expect_tx(&full[s], kABytes + kBBytes);
        tma_2d(ring + s * (kABytes + kBBytes), mw, (int)(i * kTileK), wy, &full[s]);
        tma_2d(ring + s * (kABytes + kBBytes) + kABytes, mx, xc + (int)(i * kTileK), (int)row0, &full[s]);
        issued = i + 1;
      }
      if (s_abort)  // leave no copy in flight into shared memory that another CTA may get
        for (uint32_t i = issued > (uint32_t)S ? issued - S : 0; i < issued; ++i) (void)mbar_wait(&full[i % S], (i / S) & 1u);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NT >> 3) << 17) | ((128u >> 4) << 24);  // bf16 x bf16 -> f32
      for (uint32_t i = 0; i < nk; ++i) {
        const uint32_t s = i % S;
        if (s_abort || !mbar_wait(&full[s], (i / S) & 1u)) { s_abort = 1; break; }
        tc_fence_after_sync();
        const uint64_t ad = desc_sw128(smem_u32(ring + s * (kABytes + kBBytes))), bd = desc_sw128(smem_u32(ring + s * (kABytes + kBBytes) + kABytes));
#pragma unroll
        for (uint32_t q = 0; q < kTileK / 16; ++q)
          mma_bf16(tmem, umma_desc_advance(ad, q * 32), umma_desc_advance(bd, q * 32), idesc, (i | q) != 0 ? 1u : 0u);
        umma_commit(&empty[s]);
      }
      umma_commit(&done);
    }
    grid_dependency_wait();
  } else {
    grid_dependency_wait();
    if (!mbar_wait(&done, 0)) s_abort = 1;
    tc_fence_after_sync();
    if (!s_abort) {
      const uint32_t quarter = (uint32_t)(warp & 3), j = j0 + quarter * 32 + lane;
#pragma unroll 1
      for (uint32_t c = 0; c < NT; c += 32) {
        if (row0 + c >= g.m) break;
        float v[32];
        tmem_ld32(tmem + ((quarter * 32) << 16) + c, v);
        tmem_ld_wait();
        switch (s_seg.act) {
          case ACT_SWIGLU: case ACT_GEGLU: case ACT_REGLU: finish_rows<ACT_GEGLU>(s_seg, row0 + c, g.m, j, v); break;
          case ACT_GELU: finish_rows<ACT_GELU>(s_seg, row0 + c, g.m, j, v); break;
          case ACT_SILU: finish_rows<ACT_SILU>(s_seg, row0 + c, g.m, j, v); break;
          case ACT_TANH: finish_rows<ACT_TANH>(s_seg, row0 + c, g.m, j, v); break;
          case ACT_SIGMOID: finish_rows<ACT_SIGMOID>(s_seg, row0 + c, g.m, j, v); break;
          case ACT_DECAY: finish_rows<ACT_DECAY>(s_seg, row0 + c, g.m, j, v); break;
          case ACT_FORGET: finish_rows<ACT_FORGET>(s_seg, row0 + c, g.m, j, v); break;
          default: finish_rows<ACT_NONE>(s_seg, row0 + c, g.m, j, v); break;
        }
        __syncwarp();
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (s_abort && tid == 0) atomicExch(g.status, 3);
  if (warp == 1) tmem_dealloc(tmem, NT);
}

// ---- many rows, plain f32 arithmetic -------------------------------------------------------------------

template <typename WT>
__global__ void __launch_bounds__(256) dense_simt_kernel(const Group g) {
  __shared__ float xs[16][68], ws[16][68];
  __shared__ Seg s_seg;
  const int tid = threadIdx.x;
  __shared__ bool s_any;
  grid_dependency_wait();
  grid_launch_dependents();
  if (tid == 0) {
    pick_seg(g, blockIdx.x, &s_seg);
    s_any = pick_block(&s_seg, blockIdx.x, blockIdx.y, sizeof(WT), g.x_dtype == RUAI_F32 ? 4 : 2);
  }
  __syncthreads();
  if (!s_any) return;
  const uint32_t j0 = (blockIdx.x - s_seg.tile0) * 64, row0 = blockIdx.y * 64, k = s_seg.k, n = s_seg.n;
  const uint32_t lr = tid >> 2, lk = (tid & 3) * 4, tx = tid & 15, ty = tid >> 4;
  const WT* w = reinterpret_cast<const WT*>(s_seg.w);
  float acc[4][4] = {};
  for (uint32_t k0 = 0; k0 < k; k0 += 16) {
    __syncthreads();
#pragma unroll
    for (uint32_t e = 0; e < 4; ++e) {
      const uint32_t kk = k0 + lk + e;
      xs[lk + e][lr] = (row0 + lr < g.m && kk < k) ? load_as_f32(s_seg.x, g.x_dtype, (size_t)(row0 + lr) * s_seg.ldx + kk) : 0.0f;
      ws[lk + e][lr] = (j0 + lr < n && kk < k) ? to_f32<WT>(w[(size_t)(j0 + lr) * s_seg.ldw + kk]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 16; ++kk) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[kk][ty * 4]), b = *reinterpret_cast<const float4*>(&ws[kk][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int p = 0; p < 4; ++p)
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[p][q] = fmaf(av[p], bv[q], acc[p][q]);
    }
  }
  const bool pair = is_pair(s_seg.act);
#pragma unroll
  for (int p = 0; p < 4; ++p) {
    const uint32_t row = row0 + ty * 4 + p;
    if (row >= g.m) break;
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const uint32_t j = j0 + tx * 4 + q;
      if (j >= n || (pair && (q & 1))) continue;
      finish(s_seg, row, j, acc[p][q], pair ? acc[p][(q + 1) & 3] : 0.0f);
    }
  }
}

template <typename T>
__global__ void dense_put_kernel(const float* __restrict__ src, uint32_t rows, uint32_t cols, T* __restrict__ dst, uint32_t ld, uint32_t row0, uint32_t row_step,
                                 uint32_t col0) {
  const uint32_t c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= cols) return;
  for (uint32_t r = blockIdx.y; r < rows; r += gridDim.y) dst[(size_t)(row0 + r * row_step) * ld + col0 + c] = from_f32<T>(src[(size_t)r * cols + c]);
}

typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                             const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeFn encode_fn() {
  static EncodeFn fn = [] {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult st;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &st) != cudaSuccess || st != cudaDriverEntryPointSuccess) p = nullptr;
    return (EncodeFn)p;
  }();
  return fn;
}
// A bf16 matrix of `rows` rows of k elements, `ld` apart, in boxes of box_rows x 64; out-of-range elements read as zero.
int encode(ruai_ctx* c, CUtensorMap* map, const void* base, uint32_t k, uint32_t rows, uint32_t ld, uint32_t box_rows) {
  EncodeFn fn = encode_fn();
  if (!fn) return ruai_fail(c, RUAI_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
  const cuuint64_t dims[2] = {k, rows}, strides[1] = {(cuuint64_t)ld * 2};
  const cuuint32_t box[2] = {(cuuint32_t)kTileK, box_rows}, one[2] = {1, 1};
  const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE,
                        CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return ruai_fail(c, RUAI_ERR_CUDA, "cuTensorMapEncodeTiled failed (%d) for [%u, %u] with rows %u apart", (int)r, rows, k, ld);
  return RUAI_OK;
}

// rows of W a warp works on at a time
template <typename WT> constexpr int rows_of(int mt) { return mt <= 2 && sizeof(WT) == 2 ? 8 : 4; }
template <typename WT, typename XT>
cudaError_t launch_gemv(ruai_ctx* c, const Group& g, dim3 grid, int mt, uint32_t kw) {
  switch (mt) {
    case 1: return ruai_launch(c, dense_gemv_kernel<WT, XT, 1, rows_of<WT>(1)>, grid, dim3(kVThreads), 0, true, g, kw);
    case 2: return ruai_launch(c, dense_gemv_kernel<WT, XT, 2, rows_of<WT>(2)>, grid, dim3(kVThreads), 0, true, g, kw);
    case 4: return ruai_launch(c, dense_gemv_kernel<WT, XT, 4, 4>, grid, dim3(kVThreads), 0, true, g, kw);
    default: return ruai_launch(c, dense_gemv_kernel<WT, XT, 8, 4>, grid, dim3(kVThreads), 0, true, g, kw);
  }
}

template <int NT>
cudaError_t launch_gemm(ruai_ctx* c, const Maps& maps, const Group& g, dim3 grid) {
  static bool attr_done[64] = {};
  if (!attr_done[c->ordinal & 63]) {
    cudaError_t e = cudaFuncSetAttribute(dense_gemm_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gemm_smem(NT));
    if (e != cudaSuccess) return e;
    attr_done[c->ordinal & 63] = true;
  }
  return ruai_launch(c, dense_gemm_kernel<NT>, grid, dim3(kGThreads), gemm_smem(NT), true, maps, g);
}

}  // namespace dense

int ruai_dense_alloc(ruai_ctx* c, uint32_t n, uint32_t k, uint32_t bits, ruai_qweight** out) {
  if (!n || !k || (bits != 16 && bits != 32)) return ruai_fail(c, RUAI_ERR_ARG, "unquantized weight [%u, %u] with %u bits", n, k, bits);
  ruai_qweight* w = new ruai_qweight();
  w->ctx = c; w->k = k; w->n = n; w->bits = bits; w->layout = QL_DENSE;
  w->ld = (k + 7) & ~7u;
  w->data_bytes = (size_t)n * w->ld * (bits / 8);
  cudaError_t e = cudaMalloc(&w->data, w->data_bytes);
  if (e == cudaSuccess) e = cudaMemsetAsync(w->data, 0, w->data_bytes, c->stream);
  if (e != cudaSuccess) {
    if (w->data) cudaFree(w->data);
    delete w;
    (void)cudaGetLastError();
    return ruai_fail(c, RUAI_ERR_CUDA, "unquantized weight [%u, %u]: %s", n, k, cudaGetErrorString(e));
  }
  *out = w;
  return RUAI_OK;
}

int ruai_dense_put(ruai_ctx* c, ruai_qweight* w, const float* src, uint32_t rows, uint32_t cols, uint32_t row0, uint32_t row_step, uint32_t col0) {
  if (!rows || !cols) return RUAI_OK;
  if ((size_t)row0 + (size_t)(rows - 1) * row_step >= w->n || (size_t)col0 + cols > w->k)
    return ruai_fail(c, RUAI_ERR_SHAPE, "a part [%u, %u] at (%u, %u) does not fit the weight [%u, %u]", rows, cols, row0, col0, w->n, w->k);
  const dim3 grid((cols + 255) / 256, rows < 4096 ? rows : 4096);
  if (w->bits == 16) dense::dense_put_kernel<<<grid, 256, 0, c->stream>>>(src, rows, cols, (__nv_bfloat16*)w->data, w->ld, row0, row_step, col0);
  else dense::dense_put_kernel<<<grid, 256, 0, c->stream>>>(src, rows, cols, (float*)w->data, w->ld, row0, row_step, col0);
  RUAI_CUDA(c, cudaGetLastError());
  return RUAI_OK;
}

uint32_t ruai_dense_row_tile(uint32_t m, uint32_t per_block, uint32_t bits) {
  if (m <= 16 || (m <= 128 && per_block <= 2)) return 1;  // a weight is read again for every row of its block
  if (bits == 32) return 64;
  return per_block >= 96 ? 128 : per_block >= 40 ? 64 : 32;
}

int ruai_dense_launch(ruai_ctx* c, const DenseCall* calls, int nc, int x_dtype, uint32_t m, uint32_t row_tile) {
  using namespace dense;
  if (m == 0) return RUAI_OK;
  if (nc < 1 || nc > kDenseGroupMax) return ruai_fail(c, RUAI_ERR_ARG, "a group of %d Linears (1 to %d)", nc, kDenseGroupMax);
  const uint32_t bits = calls[0].w->bits;
  Group g = {};
  g.nseg = nc; g.m = m; g.x_dtype = x_dtype; g.status = c->status;
  uint32_t k_max = 0;
  bool tma = bits == 16 && x_dtype == RUAI_BF16;
  for (int i = 0; i < nc; ++i) {
    const DenseCall& d = calls[i];
    const ruai_qweight* w = d.w;
    if (w->layout != QL_DENSE || w->bits != bits) return ruai_fail(c, RUAI_ERR_ARG, "the Linears of a group must be unquantized and of one type");
    if (d.epi.sumsq) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "unquantized Linears leave no sum of squares");
    if (is_pair(d.epi.act) && (w->n & 1)) return ruai_fail(c, RUAI_ERR_SHAPE, "a gate / up epilogue needs an even column count, got %u", w->n);
    if (d.epi.argmax_out && (nc != 1 || m > 16 || is_pair(d.epi.act))) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "fused argmax needs a Linear of its own and m <= 16");
    Seg& s = g.seg[i];
    s.w = w->data; s.x = d.x; s.out = d.out; s.bias = d.epi.bias; s.aux = d.epi.aux; s.resid = d.epi.resid;
    s.n = w->n; s.k = w->k; s.ldw = w->ld; s.ldx = d.x_ld;
    s.ldo = d.epi.out_ld ? d.epi.out_ld : (is_pair(d.epi.act) ? w->n / 2 : w->n);
    s.act = d.epi.act; s.out_dtype = d.epi.out_dtype;
    s.xdiv = 1;
    if (d.block_n) {
      if (w->n % d.block_n || (d.block_out && d.block_out > d.block_n) || d.epi.bias || d.epi.aux || d.epi.resid || d.epi.argmax_out)
        return ruai_fail(c, RUAI_ERR_ARG, "a weight of %u rows in blocks of %u has neither bias nor residual, and the blocks fill it", w->n, d.block_n);
      if ((d.table != nullptr) != (row_tile != 0) || (d.table && nc != 1)) return ruai_fail(c, RUAI_ERR_ARG, "blocks by row come alone, and with their row tile");
      s.nb = d.block_n; s.n = d.block_out ? d.block_out : d.block_n; s.xblk = d.x_block; s.oblk = d.o_block;
      s.table = d.table; s.table_early = d.table_early ? 1 : 0;
      if (d.table) s.xdiv = d.x_div;
      else if (w->n > d.block_n && ((size_t)d.x_block * (x_dtype == RUAI_F32 ? 4 : 2)) % 16) return ruai_fail(c, RUAI_ERR_ARG, "blocks of the input must start on 16 bytes");
      if (s.xdiv != 1 && row_tile != 1) return ruai_fail(c, RUAI_ERR_ARG, "rows share their input only where each is a tile of its own");
    }
    const size_t row_bytes = (size_t)d.x_ld * (x_dtype == RUAI_F32 ? 4 : 2);
    s.x_vec = ((uintptr_t)d.x % 16 == 0 && row_bytes % 16 == 0) ? 1 : 0;
    tma = tma && s.x_vec;
    k_max = w->k > k_max ? w->k : k_max;
  }
  if (calls[0].epi.argmax_out) {
    g.arg_out = calls[0].epi.argmax_out; g.arg_slots = (unsigned long long*)calls[0].epi.argmax_slots;
    g.len_ptr = calls[0].epi.len_ptr; g.len_add = calls[0].epi.len_add;
  }
  auto tiles = [&](uint32_t per) {
    uint32_t t = 0;
    for (int i = 0; i < nc; ++i) {
      Seg& q = g.seg[i];
      q.tile0 = t;
      q.tiles = (q.n + per - 1) / per;
      t += q.tiles * (q.nb && !q.table ? calls[i].w->n / q.nb : 1);
    }
    return t;
  };
  cudaError_t e;
  // f32 inputs of bf16 blocks stay on the kernel for few rows for longer: the tensor cores do not take them
  const uint32_t few = nc == 1 && g.seg[0].nb && !g.seg[0].table && x_dtype == RUAI_F32 && bits == 16 ? 64 : 16;
  if ((row_tile ? row_tile == 1 : m <= few) && x_dtype != RUAI_F16 && !(bits == 32 && x_dtype == RUAI_BF16)) {
    const int mt = row_tile ? 1 : m == 1 ? 1 : m == 2 ? 2 : m <= 4 ? 4 : 8;
    const uint32_t kw = k_max <= 256 ? 1 : k_max <= 512 ? 2 : k_max <= 1024 ? 4 : 8;
    if ((m + mt - 1) / mt > 65535) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "m too large");
    const uint32_t t = tiles((kVWarps / kw) * (bits == 32 ? rows_of<float>(mt) : rows_of<__nv_bfloat16>(mt)));
    const dim3 grid(t, (m + mt - 1) / mt);
    if (bits == 32) e = launch_gemv<float, float>(c, g, grid, mt, kw);
    else if (x_dtype == RUAI_F32) e = launch_gemv<__nv_bfloat16, float>(c, g, grid, mt, kw);
    else e = launch_gemv<__nv_bfloat16, __nv_bfloat16>(c, g, grid, mt, kw);
  } else if (tma) {
    const uint32_t t = tiles(kTileN);
    // the widest row tile that still gives every SM a CTA
    int nt = 128;
    while (nt > 32 && (m <= (uint32_t)nt / 2 || (size_t)t * ((m + nt - 1) / nt) < (size_t)c->sm_count)) nt /= 2;
    if (row_tile) {
      if (row_tile != 128 && row_tile != 64 && row_tile != 32) return ruai_fail(c, RUAI_ERR_ARG, "row tiles of %u", row_tile);
      nt = (int)row_tile;
    }
    if (t > 65535) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "n too large");
    Maps maps;
    for (int i = 0; i < nc; ++i) {
      RUAI_TRY(encode(c, &maps.w[i], g.seg[i].w, g.seg[i].k, calls[i].w->n, g.seg[i].ldw, kTileN));
      const uint32_t x_cols = g.seg[i].nb && !g.seg[i].table ? (calls[i].w->n / g.seg[i].nb - 1) * g.seg[i].xblk + g.seg[i].k : g.seg[i].k;
      RUAI_TRY(encode(c, &maps.x[i], g.seg[i].x, x_cols, m, g.seg[i].ldx, (uint32_t)nt));
    }
    for (int i = nc; i < kDenseGroupMax; ++i) { maps.w[i] = maps.w[0]; maps.x[i] = maps.x[0]; }
    const dim3 grid((m + nt - 1) / nt, t);
    e = nt == 128 ? launch_gemm<128>(c, maps, g, grid) : nt == 64 ? launch_gemm<64>(c, maps, g, grid) : launch_gemm<32>(c, maps, g, grid);
  } else {
    if (g.arg_out) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "argmax with f16 activations");
    if (row_tile && row_tile != 64) return ruai_fail(c, RUAI_ERR_ARG, "row tiles of %u", row_tile);
    const uint32_t t = tiles(64);
    if ((m + 63) / 64 > 65535) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "m too large");
    const dim3 grid(t, (m + 63) / 64);
    e = bits == 32 ? ruai_launch(c, dense_simt_kernel<float>, grid, dim3(256), 0, true, g)
                   : ruai_launch(c, dense_simt_kernel<__nv_bfloat16>, grid, dim3(256), 0, true, g);
  }
  if (e == cudaSuccess && g.arg_out) e = ruai_launch(c, dense_pick_kernel, dim3(1), dim3(kVThreads), 0, true, g);
  if (e != cudaSuccess) return ruai_fail(c, RUAI_ERR_CUDA, "unquantized Linear launch: %s", cudaGetErrorString(e));
  return RUAI_OK;
}

// An unquantized Linear for ruai_matmul_q: f32 weights [n, k] (one row per output), host or device, kept in bf16 or f32.
RUAI_API int ruai_pack_dense(ruai_ctx* c, const float* w, uint32_t n, uint32_t k, uint32_t bits, ruai_qweight** out) {
  if (!c || !w || !out) return ruai_fail(c, RUAI_ERR_ARG, "ruai_pack_dense: NULL argument");
  *out = nullptr;
  DeviceGuard guard(c->ordinal);
  ruai_qweight* q = nullptr;
  RUAI_TRY(ruai_dense_alloc(c, n, k, bits, &q));
  float* tmp = nullptr;
  int rc = RUAI_OK;
  cudaError_t e = cudaMalloc(&tmp, (size_t)n * k * sizeof(float));
  if (e == cudaSuccess) e = cudaMemcpyAsync(tmp, w, (size_t)n * k * sizeof(float), cudaMemcpyDefault, c->stream);
  if (e == cudaSuccess) rc = ruai_dense_put(c, q, tmp, n, k, 0, 1, 0);
  if (e == cudaSuccess && rc == RUAI_OK) e = cudaStreamSynchronize(c->stream);
  if (tmp) cudaFree(tmp);
  if (e != cudaSuccess) rc = ruai_fail(c, RUAI_ERR_CUDA, "ruai_pack_dense: %s", cudaGetErrorString(e));
  if (rc != RUAI_OK) { ruai_qweight_free(q); return rc; }
  *out = q;
  return RUAI_OK;
}
