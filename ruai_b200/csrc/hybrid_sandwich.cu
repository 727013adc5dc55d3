// The sandwich blocks of the decoder built from a list of layers: mixer and feed-forward one after the other, a LayerNorm
// ahead of each and another on its result before it joins the residual stream; a range of layers may run several times.
//
// A layer in a single-token step:
//   resid_norm   the last result's norm and addition, this mixer's input norm (resid_norm.cu)
//   dense group  every projection of the mixer, gates' activations fused (dense.cu)
//   latent attention, absorbed: queries through the keys' projection, head by head (dense blocks); attention of all heads
//                over the latents, with the rotation, the latent's norm and the append to the cache, and the result through
//                the values' projection (attn_latent.cu; rows it does not take: attn_span.cu and dense blocks)
//   delta rule   one kernel with convolutions, state and output norm (delta.cu)
//   dense        W_o
//   resid_norm   as above, around the feed-forward
//   dense        gate / up with the activation, then down; experts: router, choice (moe.cu), the same two by blocks
// Latent attention of eight and more tokens spreads the latents out into keys and values of every head and goes through
// attn_prefill.cu.  With many tokens the experts' tokens are sorted by expert first.
// Residual stream, norms, projections' results, scores, routing, decays and states are f32; the inputs of the matrix products
// are bf16 with 16-bit weights.
#include "hybrid_impl.cuh"

#include <algorithm>

#include "decode_ops.cuh"

namespace {

constexpr uint32_t kProjectRows = 4;   // up to here the shares of the attention are merged where the values' projection reads them
constexpr uint32_t kRouterParts = 8;
constexpr uint32_t kSpreadTokens = 8;  // from here on keys and values are spread out

bool spreads(const MixLayer& L, uint32_t T) { return L.latent() && T >= kSpreadTokens && ruai_attention_prefill_fits(L.qh(), L.vdp()); }

RotaryConfig rotary_of(const ruai_layer_config& f) {
  RotaryConfig r;
  r.rot = f.rot_dim; r.dims = f.rot_dims; r.base = f.rot_base;
  r.factor = f.yarn_factor; r.original = f.yarn_original; r.fast = f.yarn_fast; r.slow = f.yarn_slow;
  return r;
}

int pair_act_of(uint32_t act) { return act == RUAI_FF_RELU ? ACT_REGLU : act == RUAI_FF_SILU ? ACT_SWIGLU : ACT_GEGLU; }

// What the attention of a latent layer reads and writes, absorbed form: queries and values live in the latent's space.
SpanParams latent_span(const ruai_model* m, uint32_t run, uint32_t rows, uint32_t T) {
  const Hybrid* y = m->hy;
  const MixLayer& L = y->layers[y->runs[run].layer];
  const ruai_layer_config& f = L.cfg;
  SpanParams p;
  p.qkv = y->proj.as<float>();
  p.ld = L.lat_ld();
  p.k_off = f.heads * L.qh(); p.k_rot = p.k_off + f.rank;
  p.q_step = L.qh(); p.q_rot = L.dimp();
  p.k_norm = L.k_norm.as<float>(); p.eps = m->eps;
  p.T = T; p.G = 1; p.rep = f.heads; p.maps = 1; p.kd = f.rank; p.vd = f.rank; p.kdp = L.kdp(); p.vdp = L.kdp();
  p.rot = f.rot_dim; p.rotp = L.rotp();
  p.table = f.rot_dim ? y->tables[L.table].table.as<float2>() : nullptr;
  p.q_main = y->q_abs.as<float>();
  p.shared = true;
  p.cap = m->cap; p.scale = f.scale;
  p.kcache = m->layers[run].kc.as<float>();
  p.len = m->d_len.as<int32_t>();
  p.q = y->qn.as<float>();
  p.sink = L.sink.as<float>();
  p.gate = p.qkv + (size_t)rows * L.lat_ld(); p.ld_gate = f.heads;
  p.out = y->lat.p; p.out_dtype = RUAI_F32; p.out_step = L.kdp(); p.out_ld = f.heads * L.kdp();
  p.scratch = y->span_scratch.as<float>(); p.counters = y->span_counters.as<unsigned>();
  p.status = m->ctx->status;
  return p;
}

struct Calls {
  DenseCall c[kDenseGroupMax];
  int n = 0;
  DenseCall& add(const Lin& w, const void* x, uint32_t x_ld, void* out, uint32_t out_ld, int act, int dtype) {
    DenseCall& d = c[n++];
    d.w = w.w; d.x = x; d.x_ld = x_ld; d.out = out;
    d.epi.act = act; d.epi.out_dtype = dtype; d.epi.out_ld = out_ld;
    return d;
  }
};

int latent_projections(ruai_model* m, const MixLayer& L, uint32_t rows) {
  Hybrid* y = m->hy;
  float* proj = y->proj.as<float>();
  Calls k;
  k.add(L.proj[0], y->h.p, y->ldd, proj, L.lat_ld(), ACT_NONE, RUAI_F32);
  k.add(L.proj[1], y->h.p, y->ldd, proj + L.cfg.heads * L.qh(), L.lat_ld(), ACT_NONE, RUAI_F32);
  k.add(L.proj[2], y->h.p, y->ldd, proj + (size_t)rows * L.lat_ld(), L.cfg.heads, ACT_SIGMOID, RUAI_F32);
  return ruai_dense_launch(m->ctx, k.c, k.n, y->act, rows);
}
// Every head's query through its part of the keys' projection, transposed: [heads][rank].
int latent_absorb(ruai_model* m, const MixLayer& L, uint32_t rows) {
  Hybrid* y = m->hy;
  Calls k;
  DenseCall& d = k.add(L.uk_t, y->proj.p, L.lat_ld(), y->q_abs.p, L.cfg.heads * L.cfg.rank, ACT_NONE, RUAI_F32);
  d.block_n = L.cfg.rank; d.x_block = L.qh(); d.o_block = L.cfg.rank;
  return ruai_dense_launch(m->ctx, k.c, k.n, RUAI_F32, rows);
}
int latent_values(ruai_model* m, const MixLayer& L, uint32_t rows) {
  Hybrid* y = m->hy;
  Calls k;
  DenseCall& d = k.add(L.uv, y->lat.p, L.cfg.heads * L.kdp(), y->cat.p, y->ldcat, ACT_NONE, y->act);
  d.block_n = L.vdp(); d.block_out = L.cfg.vdim; d.x_block = L.kdp(); d.o_block = L.cfg.vdim;
  return ruai_dense_launch(m->ctx, k.c, k.n, RUAI_F32, rows);
}

int latent_mixer(ruai_model* m, uint32_t run, uint32_t B, uint32_t T) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  const MixLayer& L = y->layers[y->runs[run].layer];
  const ruai_layer_config& f = L.cfg;
  const uint32_t rows = B * T;
  RUAI_TRY(latent_projections(m, L, rows));
  SpanParams p = latent_span(m, run, rows, T);
  if (!spreads(L, T)) {
    RUAI_TRY(latent_absorb(m, L, rows));
    if (!ruai_attn_latent_takes(p)) {
      RUAI_TRY(ruai_attn_span(c, p, B));
      return latent_values(m, L, rows);
    }
    if (T > 1) RUAI_TRY(ruai_span_append(c, p, B));
    if (rows > kProjectRows) {
      RUAI_TRY(ruai_attn_latent(c, p, B, nullptr));
      return latent_values(m, L, rows);
    }
    LatentProjection o;
    o.w = L.uv.w; o.block_n = L.vdp(); o.rows = f.vdim; o.out = y->cat.p; o.out_ld = y->ldcat; o.out_dtype = y->act;
    return ruai_attn_latent(c, p, B, &o);
  }
  p.q_main = nullptr; p.qd = f.dim; p.qdp = L.dimp();
  RUAI_TRY(ruai_span_append(c, p, B));
  const uint32_t n = m->len + T, kw = L.kdp() + L.rotp(), ldr = hy_up8(f.rank), nk = f.heads * L.dimp(), nv = f.heads * L.vdp();
  RUAI_TRY(ruai_latent_rows(c, p.kcache, B, m->cap, kw, n, f.rank, y->lat_rows.p, ldr, y->act));
  Calls k;
  k.add(L.uk, y->lat_rows.p, ldr, y->k_all.p, nk, ACT_NONE, RUAI_F32);
  k.add(L.uv, y->lat_rows.p, ldr, y->v_all.p, nv, ACT_NONE, RUAI_F32);
  RUAI_TRY(ruai_dense_launch(c, k.c, k.n, y->act, B * n));
  AttnParams a = {};
  a.q = p.q; a.q_ld = f.heads * L.qh(); a.kcache = y->k_all.as<float>(); a.vcache = y->v_all.as<float>(); a.len = p.len; a.T = T; a.KV = f.heads;
  a.hd = L.qh(); a.vd = L.vdp(); a.vd_out = f.vdim; a.maps = 1; a.cap = n; a.scale = f.scale;
  a.k_pos = nk; a.k_head = L.dimp(); a.k_batch = (size_t)n * nk;
  a.v_pos = nv; a.v_head = L.vdp(); a.v_batch = (size_t)n * nv;
  a.hd2 = L.rotp(); a.k2 = p.kcache + L.kdp(); a.k2_pos = kw; a.k2_batch = (size_t)m->cap * kw;
  a.sink = p.sink; a.gate = p.gate; a.ld_gate = p.ld_gate;
  a.out = (float*)y->cat.p; a.out_ld = y->ldcat; a.out_dtype = y->act; a.status = c->status;
  const int took = ruai_attention_prefill(c, a, B, 1);
  if (took < 0) return RUAI_ERR_CUDA;
  return took ? RUAI_OK : model_fail(m, RUAI_ERR_UNSUPPORTED, "a step of %u sequences is too large for %u heads", B, f.heads);
}

struct DeltaRows { float *q, *k, *v, *gate, *beta, *a; uint32_t ldk, ldv, ldh; };
DeltaRows delta_rows(const Hybrid* y, const MixLayer& L, uint32_t rows) {
  DeltaRows r;
  r.ldk = hy_up4(L.cfg.kv_heads * L.cfg.dim); r.ldv = hy_up4(L.cfg.heads * L.cfg.vdim); r.ldh = hy_up4(L.cfg.heads);
  const size_t n = rows;
  r.q = y->proj.as<float>();
  r.k = r.q + n * r.ldk;
  r.v = r.k + n * r.ldk;
  r.gate = r.v + n * r.ldv;
  r.beta = r.gate + n * r.ldv;
  r.a = r.beta + n * r.ldh;
  return r;
}
int delta_projections(ruai_model* m, const MixLayer& L, uint32_t rows) {
  Hybrid* y = m->hy;
  const DeltaRows r = delta_rows(y, L, rows);
  Calls k;
  k.add(L.proj[0], y->h.p, y->ldd, r.q, r.ldk, ACT_NONE, RUAI_F32);
  k.add(L.proj[1], y->h.p, y->ldd, r.k, r.ldk, ACT_NONE, RUAI_F32);
  k.add(L.proj[2], y->h.p, y->ldd, r.v, r.ldv, ACT_NONE, RUAI_F32);
  k.add(L.proj[5], y->h.p, y->ldd, r.gate, r.ldv, ACT_SILU, RUAI_F32);
  k.add(L.proj[3], y->h.p, y->ldd, r.beta, r.ldh, ACT_SIGMOID, RUAI_F32);
  k.add(L.proj[4], y->h.p, y->ldd, r.a, r.ldh, ACT_NONE, RUAI_F32).epi.bias = L.f_bias.as<float>();
  return ruai_dense_launch(m->ctx, k.c, k.n, y->act, rows);
}
DeltaParams delta_params(const ruai_model* m, const MixLayer& L, uint32_t rows, uint32_t T) {
  const Hybrid* y = m->hy;
  const ruai_layer_config& f = L.cfg;
  const DeltaRows r = delta_rows(y, L, rows);
  DeltaParams p;
  p.q = r.q; p.k = r.k; p.v = r.v; p.a = r.a; p.beta = r.beta; p.gate = r.gate;
  p.ld_q = r.ldk; p.ld_k = r.ldk; p.ld_v = r.ldv; p.ld_a = r.ldh; p.ld_beta = r.ldh; p.ld_gate = r.ldv;
  p.conv_q = L.conv[0].as<float>(); p.conv_k = L.conv[1].as<float>(); p.conv_v = L.conv[2].as<float>();
  p.taps = f.conv; p.q_scale = 1.0f / sqrtf((float)f.dim);
  p.a_log = L.a_log.as<float>();
  p.len = m->d_len.as<int32_t>(); p.T = T; p.H = f.heads; p.G = f.kv_heads; p.dk = f.dim; p.dv = f.vdim;
  p.eps = m->eps; p.norm = L.head_norm.as<float>();
  p.out = y->cat.p; p.out_ld = y->ldcat; p.out_dtype = y->act;
  p.work = y->rec_o.as<float>();
  return p;
}
int delta_mixer(ruai_model* m, uint32_t run, uint32_t B, uint32_t T) {
  Hybrid* y = m->hy;
  MixRun& r = y->runs[run];
  const MixLayer& L = y->layers[r.layer];
  RUAI_TRY(delta_projections(m, L, B * T));
  DeltaParams p = delta_params(m, L, B * T, T);
  p.state = r.state.as<float>(); p.history = r.history.as<float>();
  return ruai_delta(m->ctx, p, B);
}

int issue_o(ruai_model* m, const MixLayer& L, uint32_t rows) {
  Calls k;
  k.add(L.o, m->hy->cat.p, m->hy->ldcat, m->hy->y.p, m->d, ACT_NONE, RUAI_F32);
  return ruai_dense_launch(m->ctx, k.c, k.n, m->hy->act, rows);
}

uint32_t expert_tile(const Hybrid* y, const ruai_layer_config& f, uint32_t rows) {
  return ruai_dense_row_tile(rows * f.top, rows * f.top / f.experts, y->act == RUAI_F32 ? 32 : 16);
}

// The experts' two products for the pairs in `chosen` (a tile of one row) or in the sorted order; results in y->y.
int issue_experts(ruai_model* m, const MixLayer& L, uint32_t rows, uint32_t tile) {
  Hybrid* y = m->hy;
  const ruai_layer_config& f = L.cfg;
  const uint32_t pairs = rows * f.top, n = tile == 1 ? pairs : ruai_route_tiles(pairs, f.experts, tile) * tile;
  const int32_t* table = (tile == 1 ? y->chosen : y->tile_expert).as<int32_t>();
  Calls up, down;
  DenseCall& u = up.add(L.up, tile == 1 ? y->h.p : y->xs.p, y->ldd, y->hid.p, y->ldff, pair_act_of(f.ff_act), y->act);
  u.block_n = 2 * f.ff; u.table = table;
  if (tile == 1) u.x_div = f.top;
  RUAI_TRY(ruai_dense_launch(m->ctx, up.c, 1, y->act, n, tile));
  DenseCall& d = down.add(L.down, y->hid.p, y->ldff, y->y.p, m->d, ACT_NONE, RUAI_F32);
  d.block_n = m->d; d.table = table; d.table_early = true;
  return ruai_dense_launch(m->ctx, down.c, 1, y->act, n, tile);
}

// The feed-forward's result into y->y; with experts the parts of every row are summed up by the next resid_norm.
int feed_forward(ruai_model* m, const MixLayer& L, uint32_t rows, ResidNormParams* next) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  const ruai_layer_config& f = L.cfg;
  if (!f.experts) {
    Calls up, down;
    up.add(L.up, y->h.p, y->ldd, y->hid.p, y->ldff, pair_act_of(f.ff_act), y->act);
    RUAI_TRY(ruai_dense_launch(c, up.c, 1, y->act, rows));
    down.add(L.down, y->hid.p, y->ldff, y->y.p, m->d, ACT_NONE, RUAI_F32);
    return ruai_dense_launch(c, down.c, 1, y->act, rows);
  }
  Calls k;
  DenseCall& r = k.add(L.router, y->h.p, y->ldd, y->scores.p, L.router_parts * f.experts, ACT_NONE, RUAI_F32);
  r.block_n = f.experts; r.x_block = m->d / L.router_parts; r.o_block = f.experts;
  RUAI_TRY(ruai_dense_launch(c, k.c, 1, y->act, rows));
  RUAI_TRY(ruai_route(c, y->scores.as<float>(), L.router_parts, L.correction.as<float>(), rows, f.experts, f.top, 1.0f, y->chosen.as<int32_t>(), y->weight.as<float>()));
  const uint32_t tile = expert_tile(y, f, rows);
  next->parts = f.top; next->part_weight = y->weight.as<float>(); next->part_row = nullptr;
  if (tile > 1) {
    RouteTiles t;
    t.place = y->place.as<int32_t>(); t.source = y->source.as<int32_t>(); t.expert = y->tile_expert.as<int32_t>();
    RUAI_TRY(ruai_route_sort(c, y->chosen.as<int32_t>(), rows, f.top, f.experts, tile, t));
    RUAI_TRY(ruai_route_gather(c, y->h.p, t.source, ruai_route_tiles(rows * f.top, f.experts, tile) * tile, y->ldd * (uint32_t)hy_act_bytes(y), y->xs.p));
    next->part_row = t.place;
  }
  return issue_experts(m, L, rows, tile);
}

NormWeights weights_of(const NormBufs& n) {
  NormWeights w;
  w.w = n.w.as<float>(); w.b = n.b.as<float>();
  return w;
}

int issue_pass_in(ruai_model* m, uint32_t rows) {
  Hybrid* y = m->hy;
  Calls k;
  k.add(y->loop_in, y->pass_in.p, y->ldpass, m->x.p, m->d, ACT_NONE, RUAI_F32);
  return ruai_dense_launch(m->ctx, k.c, 1, y->act, rows);
}

}  // namespace

int sandwich_create(ruai_model* m, HybridTensorFn add) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  const ruai_hybrid_config& cfg = y->cfg;
  const uint32_t d = cfg.width, n = cfg.num_layers;
  if (!cfg.max_positions) m->max_pos = 1u << 30;
  auto tensor = [&](const std::string& name, size_t rows, size_t cols, float std_dev, float fill = 0.0f) { add(y, name, rows, cols, std_dev, fill); };
  auto norm = [&](const std::string& name, uint32_t size) {
    tensor(name, 1, size, 0.0f, 1.0f);
    tensor(name + ".b", 1, size, 0.0f, 0.0f);
  };
  if (cfg.loop_times && (cfg.loop_start >= cfg.loop_stop || cfg.loop_stop > n))
    return ruai_fail(c, RUAI_ERR_SHAPE, "a loop over layers %u to %u of %u", cfg.loop_start, cfg.loop_stop, n);
  tensor("embed", cfg.vocab_size, d, 0.02f);
  if (cfg.loop_times) tensor("loop.in", d, 2 * (size_t)d, 0.02f);
  for (uint32_t l = 0; l < n; ++l) {
    MixLayer& L = y->layers[l];
    const ruai_layer_config& f = L.cfg;
    const std::string p = "l" + std::to_string(l) + ".", x = p + "mix.";
    if (!f.heads || !f.dim || !f.vdim) return ruai_fail(c, RUAI_ERR_SHAPE, "layer %u: heads %u, dim %u, vdim %u", l, f.heads, f.dim, f.vdim);
    const size_t hv = (size_t)f.heads * f.vdim;
    norm(p + "norm1", d);
    norm(p + "norm1b", d);
    if (f.mixer == RUAI_MIX_LATENT) {
      if (!f.rank) return ruai_fail(c, RUAI_ERR_SHAPE, "layer %u: latents of no elements", l);
      if (f.rot_dims > f.rot_dim || f.rot_dims % 2) return ruai_fail(c, RUAI_ERR_SHAPE, "layer %u: rotation of %u of %u elements", l, f.rot_dims, f.rot_dim);
      tensor(x + "q", (size_t)f.heads * (f.dim + f.rot_dim), d, 0.02f);
      tensor(x + "dkv", f.rank + f.rot_dim, d, 0.02f);
      tensor(x + "dkv.norm", 1, f.rank, 0.0f, 1.0f);
      tensor(x + "uk", (size_t)f.heads * f.dim, f.rank, 0.02f);
      tensor(x + "uv", hv, f.rank, 0.02f);
      tensor(x + "sink", 1, f.heads, 0.5f);
      tensor(x + "g", f.heads, d, 0.02f);
      const RotaryConfig r = rotary_of(f);
      L.table = 0;
      while (L.table < y->tables.size() && !(y->tables[L.table].cfg == r)) ++L.table;
      if (L.table == y->tables.size()) {
        y->tables.emplace_back();
        y->tables.back().cfg = r;
      }
    } else if (f.mixer == RUAI_MIX_DELTA) {
      if (!f.kv_heads || f.heads % f.kv_heads) return ruai_fail(c, RUAI_ERR_SHAPE, "layer %u: heads %u must be a multiple of kv_heads %u", l, f.heads, f.kv_heads);
      if (!f.conv || f.conv > (uint32_t)kConvMax) return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "layer %u: a convolution of %u taps (1 to %d)", l, f.conv, kConvMax);
      const size_t gk = (size_t)f.kv_heads * f.dim;
      for (const char* s : {"q", "k"}) { tensor(x + s, gk, d, 0.02f); tensor(x + s + ".conv", gk, f.conv, 0.5f); }
      tensor(x + "v", hv, d, 0.02f);
      tensor(x + "v.conv", hv, f.conv, 0.5f);
      tensor(x + "b", f.heads, d, 0.02f);
      tensor(x + "a", f.heads, d, 0.02f);
      tensor(x + "A_log", 1, f.heads, 0.5f);
      tensor(x + "dt_bias", 1, f.heads, 0.0f, -3.0f);
      tensor(x + "norm", 1, f.vdim, 0.0f, 1.0f);
      tensor(x + "g", hv, d, 0.02f);
    } else {
      return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "layer %u: mixer %u in a sandwich block", l, f.mixer);
    }
    tensor(x + "o", d, hv, 0.02f);
    if (!f.ff) continue;
    norm(p + "norm2", d);
    norm(p + "norm2b", d);
    const std::string q = p + "mlp.";
    if (f.ff_act > RUAI_FF_SILU) return ruai_fail(c, RUAI_ERR_ARG, "layer %u: unknown activation %u", l, f.ff_act);
    if (f.experts && (!f.top || f.top > f.experts || f.top > kRouteTopMax || f.experts > kRouteExpertsMax))
      return ruai_fail(c, RUAI_ERR_UNSUPPORTED, "layer %u: %u of %u experts (at most %u of %u)", l, f.top, f.experts, kRouteTopMax, kRouteExpertsMax);
    for (uint32_t e = 0; e < std::max(1u, f.experts); ++e) {
      const std::string s = f.experts ? q + "e" + std::to_string(e) + "." : q;
      tensor(s + "gate", f.ff, d, 0.02f);
      tensor(s + "up", f.ff, d, 0.02f);
      tensor(s + "down", d, f.ff, 0.02f);
    }
    if (f.experts) {
      tensor(q + "router", f.experts, d, 0.02f);
      tensor(q + "correction", 1, f.experts, 0.0f, 0.0f);
    }
  }
  norm("final.norm", d);
  tensor("head", cfg.vocab_size, d, 0.02f);
  auto run = [&](uint32_t l, bool first) {
    y->runs.emplace_back();
    y->runs.back().layer = l;
    y->runs.back().pass_begins = first;
  };
  const uint32_t start = cfg.loop_times ? cfg.loop_start : n, stop = cfg.loop_times ? cfg.loop_stop : n;
  for (uint32_t l = 0; l < start; ++l) run(l, false);
  for (uint32_t t = 0; t < cfg.loop_times; ++t)
    for (uint32_t l = start; l < stop; ++l) run(l, l == start);
  for (uint32_t l = stop; l < n; ++l) run(l, false);
  m->L = (uint32_t)y->runs.size();
  return RUAI_OK;
}

int sandwich_build(ruai_model* m, uint32_t bits) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  const uint32_t d = m->d;
  uint32_t cat = 0, ff = 0;
  auto norm = [&](const std::string& name, DevBuf* w, DevBuf* b) -> int {
    RUAI_TRY(hybrid_move_vec(m, name, w));
    return hybrid_move_vec(m, name + ".b", b);
  };
  for (size_t l = 0; l < y->layers.size(); ++l) {
    MixLayer& L = y->layers[l];
    const ruai_layer_config& f = L.cfg;
    const std::string p = "l" + std::to_string(l) + ".", x = p + "mix.", q = p + "mlp.";
    const uint32_t hv = f.heads * f.vdim;
    RUAI_TRY(norm(p + "norm1", &L.n1.w, &L.n1.b));
    RUAI_TRY(norm(p + "norm1b", &L.n1b.w, &L.n1b.b));
    if (L.latent()) {
      std::vector<RowPart> qp, kp, vp;
      for (uint32_t h = 0; h < f.heads; ++h) {
        const uint32_t from = h * (f.dim + f.rot_dim);
        qp.push_back({x + "q", h * L.qh(), 1, 0, from, f.dim});
        if (f.rot_dim) qp.push_back({x + "q", h * L.qh() + L.dimp(), 1, 0, from + f.dim, f.rot_dim});
        kp.push_back({x + "uk", h * L.dimp(), 1, 0, h * f.dim, f.dim});
        vp.push_back({x + "uv", h * L.vdp(), 1, 0, h * f.vdim, f.vdim});
      }
      RUAI_TRY(hybrid_build_dense(m, &L.proj[0], f.heads * L.qh(), d, bits, qp));
      RUAI_TRY(hybrid_build_dense(m, &L.proj[1], f.rank + f.rot_dim, d, bits, {{x + "dkv", 0, 1, 0}}));
      RUAI_TRY(hybrid_build_dense(m, &L.proj[2], f.heads, d, bits, {{x + "g", 0, 1, 0}}));
      const float* uk;
      RUAI_TRY(hybrid_take(m, x + "uk", &uk));
      DevBuf turned;
      int rc = turned.alloc(c, (size_t)f.heads * f.rank * f.dim * sizeof(float));
      for (uint32_t h = 0; h < f.heads && rc == RUAI_OK; ++h)
        rc = ruai_transpose_dev(c, uk + (size_t)h * f.dim * f.rank, turned.as<float>() + (size_t)h * f.dim * f.rank, f.dim, f.rank);
      if (rc == RUAI_OK) rc = ruai_dense_alloc(c, f.heads * f.rank, f.dim, bits, &L.uk_t.w);
      if (rc == RUAI_OK) rc = ruai_dense_put(c, L.uk_t.w, turned.as<float>(), f.heads * f.rank, f.dim, 0, 1, 0);
      cudaStreamSynchronize(c->stream);
      turned.release();
      RUAI_TRY(rc);
      RUAI_TRY(hybrid_build_dense(m, &L.uk, f.heads * L.dimp(), f.rank, bits, kp));
      RUAI_TRY(hybrid_build_dense(m, &L.uv, f.heads * L.vdp(), f.rank, bits, vp));
      RUAI_TRY(hybrid_move_vec(m, x + "dkv.norm", &L.k_norm));
      RUAI_TRY(hybrid_move_vec(m, x + "sink", &L.sink));
    } else {
      const uint32_t gk = f.kv_heads * f.dim;
      const char* const names[6] = {"q", "k", "v", "b", "a", "g"};
      const uint32_t sizes[6] = {gk, gk, hv, f.heads, f.heads, hv};
      for (int i = 0; i < 6; ++i) RUAI_TRY(hybrid_build_dense(m, &L.proj[i], sizes[i], d, bits, {{x + names[i], 0, 1, 0}}));
      for (int i = 0; i < 3; ++i) RUAI_TRY(hybrid_move_vec(m, x + names[i] + ".conv", &L.conv[i]));
      RUAI_TRY(hybrid_move_vec(m, x + "A_log", &L.a_log));
      RUAI_TRY(hybrid_move_vec(m, x + "dt_bias", &L.f_bias));
      RUAI_TRY(hybrid_move_vec(m, x + "norm", &L.head_norm));
    }
    RUAI_TRY(hybrid_build_dense(m, &L.o, d, hv, bits, {{x + "o", 0, 1, 0}}));
    cat = std::max(cat, hv);
    if (!f.ff) continue;
    RUAI_TRY(norm(p + "norm2", &L.n2.w, &L.n2.b));
    RUAI_TRY(norm(p + "norm2b", &L.n2b.w, &L.n2b.b));
    const uint32_t blocks = std::max(1u, f.experts);
    std::vector<RowPart> up, down;
    for (uint32_t e = 0; e < blocks; ++e) {
      const std::string s = f.experts ? q + "e" + std::to_string(e) + "." : q;
      up.push_back({s + "gate", e * 2 * f.ff, 2, 0});
      up.push_back({s + "up", e * 2 * f.ff + 1, 2, 0});
      down.push_back({s + "down", e * d, 1, 0});
    }
    RUAI_TRY(hybrid_build_dense(m, &L.up, blocks * 2 * f.ff, d, bits, up));
    RUAI_TRY(hybrid_build_dense(m, &L.down, blocks * d, f.ff, bits, down));
    if (f.experts) {
      // few columns: without parts along the inputs most SMs would have nothing to do
      L.router_parts = kRouterParts;
      while (L.router_parts > 1 && d % (8 * L.router_parts)) L.router_parts /= 2;
      const uint32_t part = d / L.router_parts;
      const float* router;
      RUAI_TRY(hybrid_take(m, q + "router", &router));
      DevBuf cut;
      int rc = cut.alloc(c, (size_t)f.experts * d * sizeof(float));
      for (uint32_t i = 0; i < L.router_parts && rc == RUAI_OK; ++i)
        if (cudaMemcpy2DAsync(cut.as<float>() + (size_t)i * f.experts * part, part * sizeof(float), router + (size_t)i * part, d * sizeof(float), part * sizeof(float), f.experts,
                              cudaMemcpyDeviceToDevice, c->stream) != cudaSuccess)
          rc = model_fail(m, RUAI_ERR_CUDA, "layer %zu: copying the router failed", l);
      if (rc == RUAI_OK) rc = ruai_dense_alloc(c, L.router_parts * f.experts, part, bits, &L.router.w);
      if (rc == RUAI_OK) rc = ruai_dense_put(c, L.router.w, cut.as<float>(), L.router_parts * f.experts, part, 0, 1, 0);
      cudaStreamSynchronize(c->stream);
      cut.release();
      RUAI_TRY(rc);
      RUAI_TRY(hybrid_drop(m, q + "router"));
      RUAI_TRY(hybrid_move_vec(m, q + "correction", &L.correction));
    }
    ff = std::max(ff, f.ff);
  }
  RUAI_TRY(hybrid_move_vec(m, "embed", &m->embed));
  RUAI_TRY(norm("final.norm", &y->final_norm, &y->final_bias));
  if (y->cfg.loop_times) RUAI_TRY(hybrid_build_dense(m, &y->loop_in, d, 2 * d, bits, {{"loop.in", 0, 1, 0}}));
  RUAI_TRY(hybrid_build_dense(m, &m->head, m->V, d, bits, {{"head", 0, 1, 0}}));
  for (RotTable& t : y->tables) {
    const std::vector<double> f = ruai_rotary_frequencies(t.cfg, &t.scale);
    RUAI_TRY(t.freq.alloc(c, f.size() * sizeof(double)));
    if (!f.empty()) RUAI_CUDA(c, cudaMemcpyAsync(t.freq.p, f.data(), f.size() * sizeof(double), cudaMemcpyHostToDevice, c->stream));
    RUAI_CUDA(c, cudaStreamSynchronize(c->stream));
  }
  y->ldd = hy_up8(d); y->ldcat = hy_up8(cat); y->ldff = hy_up8(ff); y->ldpass = hy_up8(2 * d);
  return RUAI_OK;
}

int sandwich_reserve(ruai_model* m, uint32_t rows, uint32_t B, uint32_t T) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  const size_t es = hy_act_bytes(y), r = y->rows;  // rows <= y->rows: everything is sized for the largest step so far
  size_t out = r, hid = r, abs = 0, lat = 0, work = 0, scores = 0, pairs_max = 0, sorted = 0, tiles = 0, scratch = 0, counters = 0, spread = 0, lat_ld = 0;
  for (uint32_t i = 0; i < m->L; ++i) {
    const MixLayer& L = y->layers[y->runs[i].layer];
    const ruai_layer_config& f = L.cfg;
    if (L.latent()) {
      abs = std::max(abs, (size_t)f.heads * f.rank);
      lat = std::max(lat, (size_t)f.heads * L.kdp());
      size_t n;
      if (spreads(L, T)) {
        spread = std::max(spread, (size_t)f.heads * std::max(L.dimp(), L.vdp()));
        lat_ld = std::max(lat_ld, (size_t)hy_up8(f.rank));
      } else {
        const SpanParams p = latent_span(m, i, rows, T);
        if (ruai_attn_latent_takes(p)) {
          scratch = std::max(scratch, ruai_attn_latent_scratch(p, B));
        } else {
          scratch = std::max(scratch, ruai_attn_span_scratch(p, B, &n));
          counters = std::max(counters, n);
        }
      }
    } else if (T > 1) {
      work = std::max(work, ruai_delta_work(delta_params(m, L, rows, T), (uint32_t)r, B));
    }
    if (f.ff && f.experts) {
      // the tile depends on the rows of the step: any of those that can come up
      const size_t pairs = r * f.top;
      pairs_max = std::max(pairs_max, pairs);
      scores = std::max(scores, r * L.router_parts * f.experts);
      out = std::max(out, pairs);
      for (uint32_t tile : {32u, 64u, 128u}) {
        const size_t n = ruai_route_tiles((uint32_t)pairs, f.experts, tile);
        tiles = std::max(tiles, n);
        sorted = std::max(sorted, n * tile);
      }
    }
  }
  if (sorted) { out = std::max(out, sorted); hid = std::max(hid, sorted); }
  bool synced = false;
  auto need = [&](DevBuf& b, size_t n, bool zero = false) -> int {
    if (n <= b.bytes && b.p) return RUAI_OK;
    if (!synced) {
      RUAI_CUDA(c, cudaStreamSynchronize(c->stream));
      drop_graph(m);
      synced = true;
    }
    RUAI_TRY(b.alloc(c, n));
    if (zero) RUAI_CUDA(c, cudaMemsetAsync(b.p, 0, n, c->stream));
    return RUAI_OK;
  };
  RUAI_TRY(need(y->y, out * m->d * sizeof(float)));
  RUAI_TRY(need(y->hid, hid * y->ldff * es, true));
  if (y->cfg.loop_times) RUAI_TRY(need(y->pass_in, r * y->ldpass * es));
  if (abs) RUAI_TRY(need(y->q_abs, r * abs * sizeof(float)));
  if (lat) RUAI_TRY(need(y->lat, r * lat * sizeof(float), true));
  if (work) RUAI_TRY(need(y->rec_o, work * sizeof(float)));
  if (scores) {
    RUAI_TRY(need(y->scores, scores * sizeof(float)));
    RUAI_TRY(need(y->chosen, pairs_max * sizeof(int32_t), true));
    RUAI_TRY(need(y->weight, pairs_max * sizeof(float)));
    RUAI_TRY(need(y->place, pairs_max * sizeof(int32_t)));
    RUAI_TRY(need(y->source, sorted * sizeof(int32_t)));
    RUAI_TRY(need(y->tile_expert, tiles * sizeof(int32_t)));
    RUAI_TRY(need(y->xs, sorted * y->ldd * es, true));
  }
  if (spread) {
    const size_t n = (size_t)B * m->cap;
    RUAI_TRY(need(y->lat_rows, n * lat_ld * es));
    RUAI_TRY(need(y->k_all, n * spread * sizeof(float)));
    RUAI_TRY(need(y->v_all, n * spread * sizeof(float)));
  }
  return hybrid_span_scratch(m, scratch, counters);
}

int sandwich_issue(ruai_model* m, uint32_t B, uint32_t T, const HeadRows& head, bool want_argmax) {
  Hybrid* y = m->hy;
  ruai_ctx* c = m->ctx;
  const uint32_t rows = B * T, d = m->d;
  int32_t* len = m->d_len.as<int32_t>();
  float* x = m->x.as<float>();
  const bool loop = y->cfg.loop_times != 0;
  unsigned char* beside = (unsigned char*)y->pass_in.p + (size_t)d * hy_act_bytes(y);  // the embedding's half of the passes' input
  RUAI_TRY(ruai_embed_scaled(c, m->d_ids.as<int32_t>(), m->embed.as<float>(), y->cfg.embed_scale == 0.0f ? 1.0f : y->cfg.embed_scale, rows, d, m->V, x,
                             loop ? beside : nullptr, y->ldpass, y->act, m->d_err.as<int>()));
  // what the next resid_norm has to add: nothing yet; it clears what it has used
  ResidNormParams next;
  next.x = x; next.eps = m->eps; next.rows = rows; next.d = d; next.dtype = y->act;
  const ResidNormParams plain = next;
  auto norm = [&](const NormBufs& pre) -> int {
    next.x_out = x;
    next.pre = weights_of(pre);
    next.h = y->h.p; next.h_ld = y->ldd;
    RUAI_TRY(ruai_resid_norm(c, next));
    next = plain;
    return RUAI_OK;
  };
  auto pending = [&](const NormBufs& post) {
    next.y = y->y.as<float>();
    next.post = weights_of(post);
    next.x_early = true;
  };
  for (uint32_t i = 0; i < m->L; ++i) {
    const MixRun& run = y->runs[i];
    const MixLayer& L = y->layers[run.layer];
    if (run.pass_begins) {
      next.x_out = nullptr;  // the stream is replaced
      next.cat = y->pass_in.p; next.cat_ld = y->ldpass;
      RUAI_TRY(ruai_resid_norm(c, next));
      next = plain;
      RUAI_TRY(issue_pass_in(m, rows));
    }
    RUAI_TRY(norm(L.n1));
    RUAI_TRY(L.latent() ? latent_mixer(m, i, B, T) : delta_mixer(m, i, B, T));
    RUAI_TRY(issue_o(m, L, rows));
    pending(L.n1b);
    if (L.cfg.ff) {
      RUAI_TRY(norm(L.n2));
      RUAI_TRY(feed_forward(m, L, rows, &next));
      pending(L.n2b);
    }
  }
  const uint32_t out_rows = head.count(B, T);
  if (out_rows == 0) return ruai_add_scalar(c, len, (int32_t)T);
  next.rows = out_rows;
  if (head.mode == HeadRows::LIST) next.list = m->d_rows.as<int32_t>();
  else if (head.mode == HeadRows::LAST) next.step = T;
  next.pre.w = y->final_norm.as<float>(); next.pre.b = y->final_bias.as<float>();
  next.h = y->hx.p; next.h_ld = y->ldd;
  RUAI_TRY(ruai_resid_norm(c, next));
  const bool pick = want_argmax && out_rows <= 16;
  RUAI_TRY(hybrid_issue_head(m, out_rows, pick, T));
  if (!pick) {
    RUAI_TRY(ruai_add_scalar(c, len, (int32_t)T));
    if (want_argmax) RUAI_TRY(ruai_argmax(c, m->logits.as<float>(), m->V, out_rows, m->V, m->d_ids.as<int32_t>(), 0));
  }
  return RUAI_OK;
}

int sandwich_issue_linears(ruai_model* m, uint32_t B) {
  Hybrid* y = m->hy;
  for (const MixRun& run : y->runs) {
    const MixLayer& L = y->layers[run.layer];
    if (run.pass_begins) RUAI_TRY(issue_pass_in(m, B));
    if (L.latent()) {
      RUAI_TRY(latent_projections(m, L, B));
      RUAI_TRY(latent_absorb(m, L, B));
      RUAI_TRY(latent_values(m, L, B));
    } else {
      RUAI_TRY(delta_projections(m, L, B));
    }
    RUAI_TRY(issue_o(m, L, B));
    ResidNormParams unused;
    if (L.cfg.ff) RUAI_TRY(feed_forward(m, L, B, &unused));
  }
  return RUAI_OK;
}

namespace {
// Bytes of a feed-forward's weights that a step of B tokens reads at most.
double ff_bytes(const MixLayer& L, uint32_t B) {
  const ruai_layer_config& f = L.cfg;
  if (!f.ff) return 0.0;
  const double all = L.up.bytes() + L.down.bytes();
  return f.experts ? L.router.bytes() + (double)L.correction.bytes + all * std::min(f.experts, B * f.top) / f.experts : all;
}
}  // namespace

double sandwich_linear_bytes(const ruai_model* m, uint32_t B) {
  const Hybrid* y = m->hy;
  double bytes = 0.0;
  const double es = (double)hy_act_bytes(y);
  auto lin = [&](const Lin& w) { return w.w ? w.bytes() + B * (es * w.w->k + 4.0 * w.w->n) : 0.0; };
  for (const MixRun& run : y->runs) {
    const MixLayer& L = y->layers[run.layer];
    if (run.pass_begins) bytes += lin(y->loop_in);
    for (const Lin& w : L.proj) bytes += lin(w);
    bytes += lin(L.uk_t) + lin(L.uv) + lin(L.o) + ff_bytes(L, B);
  }
  return bytes;
}

double sandwich_step_bytes(const ruai_model* m, uint32_t B, uint32_t len) {
  const Hybrid* y = m->hy;
  double w = m->head.bytes() + (double)y->final_norm.bytes * 2, per_seq = 4.0 * m->d;
  for (const MixRun& run : y->runs) {
    const MixLayer& L = y->layers[run.layer];
    const ruai_layer_config& f = L.cfg;
    if (run.pass_begins) w += y->loop_in.bytes();
    for (const Lin& l : L.proj) w += l.bytes();
    w += L.uk_t.bytes() + L.uv.bytes() + L.o.bytes() + ff_bytes(L, B);
    for (const DevBuf* b : {&L.n1.w, &L.n1.b, &L.n1b.w, &L.n1b.b, &L.n2.w, &L.n2.b, &L.n2b.w, &L.n2b.b, &L.k_norm, &L.sink, &L.f_bias, &L.a_log, &L.head_norm,
                            &L.conv[0], &L.conv[1], &L.conv[2]})
      w += (double)b->bytes;
    if (L.latent()) {
      per_seq += (double)(len + 2) * (f.rank + f.rot_dim) * 4.0;
    } else {
      per_seq += 2.0 * f.heads * f.dim * f.vdim * 4.0 + (double)f.conv * (2.0 * f.kv_heads * f.dim + f.heads * f.vdim) * 4.0;
    }
  }
  return w + B * per_seq;
}
